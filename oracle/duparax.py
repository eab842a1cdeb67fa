"""Plain, slow restatement of the Duparax layer equations in torch on the CPU -- TEST INFRASTRUCTURE ONLY.

One function per mechanism, written token by token (explicit loops over positions, heads, blocks and experts; no paging, no
batching, no key ranges, no stacked projections, no chunked scans): the opposite route from the product kernels in
lmdeploy_b200/csrc/hybrid, with which it shares no code.  `dt` is the dtype everything runs in (float64 by default).

Notation: n tokens of one sequence, W model width; weights are stored [out, in] and applied as x @ W.T; rms(x) is x divided by
sqrt(mean(x^2) + eps).

A layer norms what each sublayer READS and what it GIVES:
    x <- x + rms(mixer(rms(x) * n1)) * n1b,    x <- x + rms(ff(rms(x) * n2)) * n2b.
Two kinds of mixer:
  parallel -- two mixers on the same input, (rms(left) * w_l + rms(right) * w_r) / 2:
      left:  softmax attention over all earlier positions, grouped key/value heads, biased projections, no rotation; a query at
             position p grows by 1 + coef * ln(1 + floor((p + 1) / every));
      right: gated linear attention: per head a [dim, vdim] matrix S, decayed per key channel by sigmoid(z)^(1/tau) with z a low-rank
             function of the token; read AFTER the token's own key and value have joined it; unit norm per head, silu gate.
  rglru    -- two branches: gelu(y) and a causal convolution u; u drives a real-gated diagonal recurrence whose decay and input
             gates are block-diagonal functions of u; the state times gelu(y) is projected.
Feed-forward: gated silu (dense), or routed experts of that form (softmax over the chosen logits) beside a shared one."""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + torch.clamp(x, min=0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def query_growth(position, q_temp):
    """The factor on a query at `position`; q_temp None: 1."""
    if q_temp is None:
        return 1.0
    return 1.0 + q_temp["coef"] * math.log(math.floor((position + 1) / q_temp["every"]) + 1)


def new_attention_state(m, dt=torch.float64):
    G = m["kv_heads"]
    return dict(k=torch.zeros(0, G, m["dim"], dtype=dt), v=torch.zeros(0, G, m["vdim"], dtype=dt))


def attention(h, p, m, positions, state):
    """The left mixer: h [n, W]; state holds the keys and values of earlier positions."""
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    out = torch.zeros(h.shape[0], H * V, dtype=h.dtype)
    for t in range(h.shape[0]):
        q = (h[t] @ p["q"].T + p["q.b"]).reshape(H, D) * query_growth(positions[t], m.get("q_temp"))
        k = (h[t] @ p["k"].T + p["k.b"]).reshape(G, D)
        v = (h[t] @ p["v"].T + p["v.b"]).reshape(G, V)
        state["k"] = torch.cat([state["k"], k[None]], 0)
        state["v"] = torch.cat([state["v"], v[None]], 0)
        for a in range(H):
            g = a // (H // G)
            weights = torch.softmax(state["k"][:, g] @ q[a] * m["scale"], 0)
            out[t, a * V:(a + 1) * V] = weights @ state["v"][:, g]
    return out @ p["o"].T


def new_linear_state(m, dt=torch.float64):
    return dict(S=torch.zeros(m["heads"], m["dim"], m["vdim"], dtype=dt))


def channel_decays(h_t, p, m):
    """[heads, dim] decays of one token: sigmoid(z)^(1/tau)."""
    z = (h_t @ p["a1"].T) @ p["a2"].T + p["a2.b"]
    return sigmoid(z).pow(1.0 / m["tau"]).reshape(m["heads"], m["dim"])


def gated_linear_attention(h, p, m, eps, state):
    """The right mixer; state['S'] [heads, dim, vdim]."""
    H, D, V = m["heads"], m["dim"], m["vdim"]
    out = torch.zeros(h.shape[0], H * V, dtype=h.dtype)
    for t in range(h.shape[0]):
        q = (h[t] @ p["q"].T).reshape(H, D) * D ** -0.5
        k = (h[t] @ p["k"].T).reshape(H, D)
        v = (h[t] @ p["v"].T).reshape(H, V)
        alpha = channel_decays(h[t], p, m)
        o = torch.zeros(H, V, dtype=h.dtype)
        for a in range(H):
            state["S"][a] = alpha[a][:, None] * state["S"][a] + torch.outer(k[a], v[a])
            o[a] = state["S"][a].T @ q[a]
        out[t] = (unit_rms(o, eps) * p["norm"]).reshape(-1) * silu(h[t] @ p["g"].T)
    return out @ p["o"].T


def side_by_side(h, p, m, eps, positions, state):
    left = attention(h, sub(p, "left."), m["left"], positions, state["left"])
    right = gated_linear_attention(h, sub(p, "right."), m["right"], eps, state["right"])
    return 0.5 * (unit_rms(left, eps) * p["left.out"] + unit_rms(right, eps) * p["right.out"])


def new_rglru_state(m, dt=torch.float64):
    return dict(S=torch.zeros(m["width"], dtype=dt), conv=torch.zeros(m["conv"] - 1, m["width"], dtype=dt))


def rglru_gates(u_t, p, blocks):
    """(r, i) of one token: every block's two square maps over its own part of u."""
    size = u_t.shape[0] // blocks
    r, i = torch.zeros_like(u_t), torch.zeros_like(u_t)
    for b in range(blocks):
        part = slice(b * size, (b + 1) * size)
        r[part] = sigmoid(p["ra"][b] @ u_t[part] + p["ra.b"][b])
        i[part] = sigmoid(p["ri"][b] @ u_t[part] + p["ri.b"][b])
    return r, i


def rglru(h, p, m, state):
    """state['conv']: the last taps - 1 inputs of the convolution, oldest first; state['S'] [width]."""
    taps = m["conv"]
    out = torch.zeros(h.shape[0], m["width"], dtype=h.dtype)
    for t in range(h.shape[0]):
        y = gelu_tanh(h[t] @ p["y"].T + p["y.b"])
        recent = torch.cat([state["conv"], (h[t] @ p["x"].T + p["x.b"])[None]], 0)            # [taps, width]
        state["conv"] = recent[1:]
        u = p["conv.b"] + sum(p["conv"][:, j] * recent[j] for j in range(taps))
        r, i = rglru_gates(u, p, m["blocks"])
        a = torch.exp(-8.0 * r * softplus(p["lam"]))
        state["S"] = a * state["S"] + torch.sqrt(1.0 - a * a) * i * u
        out[t] = state["S"] * y
    return out @ p["o"].T


def gated_ff(h, p):
    return (silu(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def route(h_t, p, f):
    """One token -> [(expert, weight)]: the largest logits, softmax over the chosen ones only."""
    z = h_t @ p["router"].T + p["router.b"]
    chosen = sorted(range(f["router"]["experts"]), key=lambda e: (-float(z[e]), e))[:f["router"]["top"]]
    weights = torch.softmax(z[chosen], 0)
    return [(e, weights[j]) for j, e in enumerate(chosen)]


def routed_ff(h, p, f):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in route(h[t], p, f):
            out[t] += weight * gated_ff(h[t], sub(p, f"e{e}."))
    if f.get("shared"):
        out = out + gated_ff(h, sub(p, "shared."))
    return out


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


class Decoder:
    """A Duparax decoder over one sequence: forward(tokens) continues from what earlier calls left."""

    def __init__(self, cfg, tensors, dt=torch.float64):
        self.cfg, self.dt = cfg, dt
        self.w = {k: v.to(dt) for k, v in tensors.items()}
        self.state = []
        for e in cfg["layers"]:
            m = e["mixer"]
            if e["type"] == "parallel":
                self.state.append(dict(left=new_attention_state(m["left"], dt), right=new_linear_state(m["right"], dt)))
            elif e["type"] == "rglru":
                self.state.append(new_rglru_state(m, dt))
            else:
                raise NotImplementedError(e["type"])
        self.pos = 0

    def forward(self, tokens, trace=None):
        """-> logits [n, vocab]; trace (a list) receives the stream after every layer."""
        cfg, w = self.cfg, self.w
        eps = cfg["norm"]["eps"]
        positions = list(range(self.pos, self.pos + len(tokens)))
        self.pos += len(tokens)
        x = torch.stack([w["embed"][t] for t in tokens])
        for i, e in enumerate(cfg["layers"]):
            p = f"l{i}."
            h = unit_rms(x, eps) * w[p + "norm1"]
            mix = sub(w, p + "mix.")
            if e["type"] == "parallel":
                y = side_by_side(h, mix, e["mixer"], eps, positions, self.state[i])
            else:
                y = rglru(h, mix, e["mixer"], self.state[i])
            x = x + unit_rms(y, eps) * w[p + "norm1b"]
            f = e.get("mlp")
            if f is not None:
                h = unit_rms(x, eps) * w[p + "norm2"]
                mlp = sub(w, p + "mlp.")
                y = gated_ff(h, mlp) if f["kind"] == "dense" else routed_ff(h, mlp, f)
                x = x + unit_rms(y, eps) * w[p + "norm2b"]
            if trace is not None:
                trace.append(x.clone())
        return (unit_rms(x, eps) * w["final.norm"]) @ w["head"].T * cfg.get("logit_scale", 1.0)

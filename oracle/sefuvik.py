"""Plain, slow restatement of the Sefuvik layer equations in torch on the CPU -- TEST INFRASTRUCTURE ONLY.

One function per mechanism, written token by token (explicit loops over positions, heads, streams and keys; no paging, no
batching, no key ranges, no stacked projections, no scans by tiles): the opposite route from the product kernels in
lmdeploy_b200/csrc/hybrid, with which it shares no code.  `dt` is the dtype everything runs in (float64 by default).

Notation: n tokens of one sequence, W model width; weights are stored [out, in] and applied as x @ W.T; rms(x) is x divided by
sqrt(mean(x^2) + eps).  The model's norms multiply by 1 + w.

The residual is s parallel streams.  A sublayer f with its vectors a, c [s] and matrix M [s, s] (from, to):
    u = sum_i a_i x_i;   y = ls * f(rms(u) (1 + w));   x_j <- sum_i M_ij x_i + c_j y      (all at once)
Three kinds of mixer:
  attention -- differential: two softmax maps per head over a sliding window plus the sequence's first tokens, subtracted with a
               learned factor, unit norm per head; biased projections, no rotation;
  retention -- linear attention with a fixed decay per head on rotated queries and keys, unit norm per head, silu gate;
  parallel  -- a weighted sum of two: softmax attention within chunks (rotation, a sink in the denominator, a gate per column)
               and the gated delta rule (short convolutions, unit queries and keys, a decay per key channel).
Feed-forward: down(gelu(gate) * up)."""
import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + torch.clamp(x, min=0.0)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_halves(x, position, rot):
    """x [..., dim]: dimension i turns with dimension i + dims/2, i < dims/2, by position * base^(-2i/dims); the rest stays."""
    half = rot["dims"] // 2
    out = x.clone()
    for i in range(half):
        a = position * rot["base"] ** (-2.0 * i / rot["dims"])
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * math.cos(a) - v * math.sin(a)
        out[..., i + half] = v * math.cos(a) + u * math.sin(a)
    return out


# ------------------------------------------------------------------------------------------------ differential attention
def new_differential_state(m, dt=torch.float64):
    G = m["kv_heads"]
    return dict(k=torch.zeros(0, G, 2, m["dim"], dtype=dt), v=torch.zeros(0, G, m["vdim"], dtype=dt))


def window_keys(i, size, keep_first):
    """The positions that position i sees: the last `size` ones, its own included, and the sequence's first `keep_first`."""
    return [j for j in range(i + 1) if i - j < size or j < keep_first]


def subtraction_factor(p, m):
    return torch.exp((p["lq1"] * p["lk1"]).sum()) - torch.exp((p["lq2"] * p["lk2"]).sum()) + m["diff"]


def differential_attention(h, p, m, eps, positions, state):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mask = m.get("mask") or {}
    lam = subtraction_factor(p, m)
    out = torch.zeros(h.shape[0], H * V, dtype=h.dtype)
    for t in range(h.shape[0]):
        q = (h[t] @ p["q"].T + p["q.b"]).reshape(H, 2, D)
        k = (h[t] @ p["k"].T + p["k.b"]).reshape(G, 2, D)
        v = (h[t] @ p["v"].T + p["v.b"]).reshape(G, V)
        state["k"] = torch.cat([state["k"], k[None]], 0)
        state["v"] = torch.cat([state["v"], v[None]], 0)
        seen = window_keys(positions[t], mask.get("size") or positions[t] + 1, mask.get("keep_first") or 0)
        for a in range(H):
            g = a // (H // G)
            maps = [torch.softmax(state["k"][seen, g, b] @ q[a, b] * m["scale"], 0) @ state["v"][seen, g] for b in range(2)]
            out[t, a * V:(a + 1) * V] = unit_rms(maps[0] - lam * maps[1], eps) * (1.0 - m["diff"])
    return out @ p["o"].T


# ------------------------------------------------------------------------------------------------ retention
def new_retention_state(m, dt=torch.float64):
    return dict(S=torch.zeros(m["heads"], m["dim"], m["vdim"], dtype=dt))


def retention(h, p, m, eps, positions, state):
    H, D, V = m["heads"], m["dim"], m["vdim"]
    out = torch.zeros(h.shape[0], H * V, dtype=h.dtype)
    for t in range(h.shape[0]):
        q = rotate_halves((h[t] @ p["q"].T).reshape(H, D), positions[t], m["rot"])
        k = rotate_halves((h[t] @ p["k"].T).reshape(H, D), positions[t], m["rot"]) * D ** -0.5
        v = (h[t] @ p["v"].T).reshape(H, V)
        o = torch.zeros(H, V, dtype=h.dtype)
        for a in range(H):
            state["S"][a] = m["decay"][a] * state["S"][a] + torch.outer(k[a], v[a])
            o[a] = state["S"][a].T @ q[a]
        out[t] = unit_rms(o, eps).reshape(-1) * silu(h[t] @ p["g"].T)
    return out @ p["o"].T


# ------------------------------------------------------------------------------------------------ chunked attention with a sink
def new_chunked_state(m, dt=torch.float64):
    G = m["kv_heads"]
    return dict(k=torch.zeros(0, G, m["dim"], dtype=dt), v=torch.zeros(0, G, m["vdim"], dtype=dt))


def chunk_keys(i, size):
    """The positions that position i sees: those of its own chunk up to itself."""
    return [j for j in range(i + 1) if j // size == i // size]


def chunked_attention(h, p, m, positions, state):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    size = (m.get("mask") or {}).get("size")
    out = torch.zeros(h.shape[0], H * V, dtype=h.dtype)
    for t in range(h.shape[0]):
        q = rotate_halves((h[t] @ p["q"].T).reshape(H, D), positions[t], m["rot"])
        k = rotate_halves((h[t] @ p["k"].T).reshape(G, D), positions[t], m["rot"])
        state["k"] = torch.cat([state["k"], k[None]], 0)
        state["v"] = torch.cat([state["v"], (h[t] @ p["v"].T).reshape(1, G, V)], 0)
        seen = chunk_keys(positions[t], size or positions[t] + 1)
        for a in range(H):
            g = a // (H // G)
            scores = torch.cat([state["k"][seen, g] @ q[a] * m["scale"], p["sink"][a:a + 1]])
            weights = torch.softmax(scores, 0)[:-1]
            out[t, a * V:(a + 1) * V] = weights @ state["v"][seen, g]
        out[t] *= sigmoid(h[t] @ p["g"].T)
    return out @ p["o"].T


# ------------------------------------------------------------------------------------------------ gated delta rule
def new_delta_state(m, dt=torch.float64):
    K, V, past = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["conv"] - 1
    return dict(S=torch.zeros(m["heads"], m["dim"], m["vdim"], dtype=dt), q=torch.zeros(past, K, dtype=dt), k=torch.zeros(past, K, dtype=dt),
                v=torch.zeros(past, V, dtype=dt))


def short_convolution(x_t, w, past):
    """x_t [channels] joins its predecessors past [taps - 1, channels] -> (silu of the weighted sum, the new past)."""
    recent = torch.cat([past, x_t[None]], 0)
    return silu(sum(w[:, j] * recent[j] for j in range(w.shape[1]))), recent[1:]


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_decays(h_t, p, m):
    """[heads, dim] decays of one token."""
    z = (h_t @ p["a1"].T) @ p["a2"].T + p["dt_bias"]
    return torch.exp(-torch.exp(p["A_log"])[:, None] * softplus(z).reshape(m["heads"], m["dim"]))


def delta_update(S, decay, k, v, beta):
    """One head's matrix [dim, vdim] after one token."""
    S = decay[:, None] * S
    return S + torch.outer(k, beta * (v - S.T @ k))


def gated_delta_rule(h, p, m, eps, state):
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    out = torch.zeros(h.shape[0], H * V, dtype=h.dtype)
    for t in range(h.shape[0]):
        qkv = {}
        for c in "qkv":
            qkv[c], state[c] = short_convolution(h[t] @ p[c].T, p[c + ".conv"], state[c])
        q = unit_vector(qkv["q"].reshape(G, D)) * D ** -0.5
        k = unit_vector(qkv["k"].reshape(G, D))
        v = qkv["v"].reshape(H, V)
        beta = sigmoid(h[t] @ p["b"].T)
        decay = channel_decays(h[t], p, m)
        o = torch.zeros(H, V, dtype=h.dtype)
        for a in range(H):
            g = a // (H // G)
            state["S"][a] = delta_update(state["S"][a], decay[a], k[g], v[a], beta[a])
            o[a] = state["S"][a].T @ q[g]
        gate = sigmoid((h[t] @ p["g1"].T) @ p["g2"].T)
        out[t] = (unit_rms(o, eps) * p["norm"]).reshape(-1) * gate
    return out @ p["o"].T


def side_by_side(h, p, m, eps, positions, state):
    left = chunked_attention(h, sub(p, "left."), m["left"], positions, state["left"])
    right = gated_delta_rule(h, sub(p, "right."), m["right"], eps, state["right"])
    return m["left_scale"] * left + m["right_scale"] * right


# ------------------------------------------------------------------------------------------------ feed-forward, streams
def gated_ff(h, p):
    return (gelu_tanh(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def read_streams(xs, a):
    """xs: list of s tensors [n, W] -> their weighted sum."""
    return sum(a[i] * xs[i] for i in range(len(xs)))


def write_streams(xs, M, c, y):
    return [sum(M[i, j] * xs[i] for i in range(len(xs))) + c[j] * y for j in range(len(xs))]


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


class Decoder:
    """A Sefuvik decoder over one sequence: forward(tokens) continues from what earlier calls left."""

    def __init__(self, cfg, tensors, dt=torch.float64):
        self.cfg, self.dt = cfg, dt
        self.w = {k: v.to(dt) for k, v in tensors.items()}
        self.state = []
        for e in cfg["layers"]:
            m = e["mixer"]
            if e["type"] == "attention":
                self.state.append(new_differential_state(m, dt))
            elif e["type"] == "retention":
                self.state.append(new_retention_state(m, dt))
            elif e["type"] == "parallel":
                self.state.append(dict(left=new_chunked_state(m["left"], dt), right=new_delta_state(m["right"], dt)))
            else:
                raise NotImplementedError(e["type"])
        self.pos = 0

    def mixer(self, i, h, positions):
        e, eps = self.cfg["layers"][i], self.cfg["norm"]["eps"]
        p = sub(self.w, f"l{i}.mix.")
        if e["type"] == "attention":
            return differential_attention(h, p, e["mixer"], eps, positions, self.state[i])
        if e["type"] == "retention":
            return retention(h, p, e["mixer"], eps, positions, self.state[i])
        return side_by_side(h, p, e["mixer"], eps, positions, self.state[i])

    def forward(self, tokens, trace=None):
        """-> logits [n, vocab]; trace (a list) receives the sum of the streams after every layer."""
        cfg, w = self.cfg, self.w
        eps = cfg["norm"]["eps"]
        positions = list(range(self.pos, self.pos + len(tokens)))
        self.pos += len(tokens)
        x = norm(torch.stack([w["embed"][t] for t in tokens]), w["embed.norm"], eps)
        xs = [x.clone() for _ in range(cfg["streams"])]
        for i, e in enumerate(cfg["layers"]):
            p = f"l{i}."
            for q in (1, 2) if e.get("mlp") is not None else (1,):
                hc = sub(w, p + f"hc{q}.")
                h = norm(read_streams(xs, hc["in"]), w[p + f"norm{q}"], eps)
                y = self.mixer(i, h, positions) if q == 1 else gated_ff(h, sub(w, p + "mlp."))
                xs = write_streams(xs, hc["mix"], hc["out"], y * w[p + f"ls{q}"])
            if trace is not None:
                trace.append(sum(xs))
        return norm(sum(xs), w["final.norm"], eps) @ w["embed"].T

"""Scenarios every engine serving a Duparax decoder must pass, whatever runs its operators: `make(cfg, tensors, **kw)` builds
the engine (duparax_cases.build_engine with a device, dtype and library chosen by the caller), `tol` bounds
hybrid_cases.rel_error against the float64 oracle.  Run on the CPU through the numpy stand-in (tests/test_duparax_cpu.py: host
logic -- pages, slots, row addressing, scheduling, state offsets) and on a GPU through the CUDA kernels (tests/test_duparax_gpu.py)."""
import ctypes as C

import numpy as np
import torch

import duparax_cases as DC
from fogizen_scenarios import _close, _in_portions, _sub64
from oracle import duparax as D


def _check(got, want, tol, what, make=None):
    """Every position within tol; for an engine whose projections are rounded (make.all_experts) one position in fifty may reach 2.5 tol:
    a unit norm over a head's few channels now and then divides by a small root mean square, which multiplies the rounding of what
    it norms at that lone position.  (A fault of a page, a slot or a state moves all positions after it.)"""
    err = DC.rel_error(got, want)
    lone = max(1, len(err) // 50) if getattr(make, "all_experts", False) else 0
    worst = np.sort(err)[::-1]
    assert worst[0] <= (2.5 * tol if lone else tol), f"{what}: relative error {err.max():.3g} at position {int(err.argmax())} (bound {tol})"
    assert len(err) <= lone or worst[lone] <= tol, f"{what}: relative error {worst[lone]:.3g} at {lone + 1} positions (bound {tol})"


def _config(make, **kw):
    """DC.config for an engine built by `make`.  Rounding flips a router's choice wherever two logits are close, which moves a
    position's logits by their whole size without being a fault; so engines that say so (make.all_experts) get routers that take ALL
    their experts -- still weighted by the softmax of their logits --, and the choice itself is tested on exact inputs (router_alone)
    and in float32 everywhere.  Their attention scores are a third of the others': a softmax over scores of tens multiplies the
    rounding of queries and keys by as much (sharp scores are tested on exact inputs, marked_keys_and_growing_queries)."""
    cfg = DC.config(**kw)
    if getattr(make, "all_experts", False):
        for entry in cfg["layers"]:
            if entry["type"] == "parallel":
                entry["mixer"]["left"] = dict(entry["mixer"]["left"], scale=0.3 * entry["mixer"]["left"]["scale"])
            if entry["mlp"] is not None and entry["mlp"]["kind"] == "moe":
                entry["mlp"]["router"]["top"] = entry["mlp"]["router"]["experts"]
    return cfg


def _weights(make, cfg, seed=0):
    """DC.random_tensors for an engine built by `make`.  Where a head of the gated linear attention has seen one token, its unit norm
    leaves the SIGN of q.k times a unit value: with q.k near zero rounding decides it.  Engines whose projections are rounded
    (make.all_experts) get keys that lie along the queries; float32 engines take the weights as they come."""
    w = DC.random_tensors(cfg, seed=seed)
    if getattr(make, "all_experts", False):
        for name in list(w):
            if name.endswith("mix.right.k"):
                w[name] = (w[name[:-1] + "q"] + 0.25 * w[name]).to(torch.bfloat16).float()
    return w


def _run(make, tol, lengths, schedule, seed, what, cfg=None, **kw):
    """A schedule against the oracle on every request's whole token list -> the engine."""
    cfg = cfg or _config(make)
    w = _weights(make, cfg, seed=seed)
    P = DC.prompts_for(cfg, lengths)
    eng = make(cfg, w, **kw)
    got = DC.replay(eng, P, schedule)
    want = {k: DC.oracle_logits(cfg, w, P[k]) for k in P}
    for k, v in got.items():
        _check(v, want[k.split("#")[0]], tol, f"{what} {k}", make)
    return eng


def whole_prompt(make, tol):
    """Whole prompts: longer than two pages, a single token, a few tokens."""
    _run(make, tol, {"a": 150, "b": 1, "c": 5}, [[("a", 150)], [("b", 1)], [("c", 5)]], 0, "whole prompt")


def layer_by_layer(make, tol):
    """The residual stream after every layer against the oracle's."""
    cfg = _config(make)
    w = _weights(make, cfg, seed=2)
    P = DC.prompts_for(cfg, {"a": 80})
    eng = make(cfg, w)
    eng.layer_trace = []
    DC.replay(eng, P, [[("a", 80)]])
    want = []
    DC.oracle_logits(cfg, w, P["a"], trace=want)
    assert len(eng.layer_trace) == len(want) == 5
    for r, (g, x) in enumerate(zip(eng.layer_trace, want)):
        err = float((g.double().cpu() - x).abs().max() / x.abs().max())
        assert err <= tol, f"stream after layer {r}: {err:.3g} of its largest value (bound {tol})"


def prefill_then_decode(make, tol, n=200, tail=120):
    """Most of a prompt in one step, the rest token by token: decoded tokens cross page borders (127 -> 128, 191 -> 192) and the
    places where the queries grow; both recurrences are carried over more than a hundred single-token steps."""
    _run(make, tol, {"a": n}, [[("a", n - tail)]] + [[("a", 1)]] * tail, 3, "prefill then decode")


def token_by_token(make, tol, n=70):
    """Every token alone from the first: zero states, zeros before the convolution, a lone key."""
    _run(make, tol, {"a": n}, [[("a", 1)]] * n, 4, "token by token")


def portions(make, tol):
    """Portions of several sizes down to one and two tokens (shorter than the convolution), cut inside pages and at their borders
    and around row counts where the scan's tiles end."""
    cuts = [2, 3, 1, 2, 29, 13, 14, 2, 1, 33, 28, 2, 64, 5, 9, 2, 129, 7, 2]
    _run(make, tol, {"a": sum(cuts)}, [[("a", c)] for c in cuts], 5, "portions", blocks=8)


def unequal_batch(make, tol):
    """Requests of unequal length in one batch -- portions beside single tokens -- against each alone."""
    sched = [[("a", 30), ("b", 3)], [("b", 1), ("c", 64), ("a", 2)], [("a", 50), ("d", 2), ("c", 1), ("b", 1)],
             [("c", 1), ("a", 1), ("b", 2)], [("a", 7)]]
    _run(make, tol, {"a": 90, "b": 7, "c": 66, "d": 2}, sched, 6, "batched")


def left_out_and_resumed(make, tol):
    """A request sits steps out while others run and another takes a slot beside it; it goes on from its pages and state."""
    sched = [[("a", 40), ("b", 2)], [("b", 9)], [("c", 70), ("b", 1)], [("b", 3), ("c", 1)], [("a", 1)], [("c", 4)], [("a", 30), ("b", 5)]]
    _run(make, tol, {"a": 71, "b": 20, "c": 75}, sched, 16, "resumed")


def reuse_of_pages_and_slots(make, tol):
    """A pool of 3 pages and 2 state slots serves requests one after another and side by side: every page and slot is handed
    out again, and a request repeated in a used slot (whose states another request left) gives what it gave in a fresh one."""
    sched = [[("a", 64), ("b", 20)], [("a", 36), ("c", 10)], [("c", 54), ("b#2", 5)], [("b#2", 15), ("a#2", 30)], [("a#2", 70)],
             [("c#2", 64), ("b#3", 20)]]
    eng = _run(make, tol, {"a": 100, "b": 20, "c": 64}, sched, 7, "reuse", blocks=3, max_batch=2)
    assert eng.scheduler.alloc.num_free == 3 and sorted(eng.scheduler.slots) == [0, 1]


def other_sizes(make, tol):
    """Sizes that a given model may make equal or 1: one layer of either kind; one head on each side; as many key/value heads as
    heads; value heads wider and narrower than key heads on both sides; no query growth, growth at every position, growth later than
    the prompt, a fractional step; tau 1; inner decay size 1 and an odd one; recurrent heads narrower than a warp, wider than 128
    channels, with states that are not 16-byte aligned; one block, as many blocks as channels, odd channel counts; 1 tap, more than 4
    taps; one expert, all experts chosen, no shared expert, a shared expert of another size; no feed-forward; logit scale 1."""
    P, L, R, G, E, F = DC.pair, DC.left, DC.right, DC.rglru, DC.moe, DC.dense
    stacks = [
        dict(layers=[P(L(heads=1, kv_heads=1, dim=4, vdim=4, q_temp=None), R(heads=1, dim=4, vdim=4, rank=1, tau=1.0))], width=16, vocab=9,
             logit_scale=1.0),
        dict(layers=[G(width=7, blocks=1, conv=1)], width=16, vocab=9),
        dict(layers=[G(width=16, blocks=16, conv=7, mlp=E(experts=1, top=1, ff=8, shared=5)),
                     P(L(heads=5, kv_heads=5, dim=6, vdim=3, q_temp=(0.5, 1)), R(heads=1, dim=40, vdim=3, rank=2), mlp=F(ff=7))], width=16, vocab=9),
        dict(layers=[P(L(heads=8, kv_heads=2, dim=4, vdim=9, q_temp=(2.0, 1000)), R(heads=6, dim=3, vdim=70, rank=4), mlp=E(experts=4, top=4, ff=12, shared=0)),
                     P(mlp=F(ff=9)), G(width=90, blocks=2, conv=3, mlp=E(experts=8, top=1, ff=10, shared=30))], width=40, vocab=33),
        # a width that leaves the recurrent states unaligned for 16-byte reads and rows for vector accesses; heads wider than 128 channels
        dict(layers=[P(L(q_temp=(0.3, 2.5)), R(heads=1, dim=130, vdim=34, rank=3)), G(width=33, blocks=3, conv=2),
                     P(r=R(heads=2, dim=36, vdim=36, rank=7, tau=9.5), mlp=F(ff=9))], width=33, vocab=20),
    ]
    for k, kw in enumerate(stacks):
        _run(make, tol, {"a": 131, "b": 4}, [[("a", 3)], [("a", 62), ("b", 2)], [("a", 1), ("b", 1)], [("a", 1)], [("a", 62), ("b", 1)], [("a", 1)],
                                             [("a", 1)]], 10 + k, f"sizes {k}", cfg=_config(make, **kw))


def wider_sizes(make, tol):
    """Sizes of the order of a real layer's heads: 16 query heads on 2 key/value heads, head dimensions of 64 and 128 (16-byte
    key reads) and an odd one (scalar reads), wide value heads, recurrent heads of 64 and 128 channels, recurrent branches wider and
    narrower than the model, expert widths that are and are not multiples of eight, prompts long enough for grouped expert GEMMs, key
    ranges and several tiles of the scan."""
    P, L, R, G, E, F = DC.pair, DC.left, DC.right, DC.rglru, DC.moe, DC.dense
    stacks = [
        dict(layers=[P(L(heads=16, kv_heads=2, dim=64, vdim=64, scale=0.125, q_temp=(0.3, 128)), R(heads=4, dim=64, vdim=64, rank=16),
                       mlp=E(experts=4, top=2, ff=64, shared=96)),
                     G(width=256, blocks=4, conv=4, mlp=F(ff=160)),
                     P(L(heads=4, kv_heads=4, dim=128, vdim=32, scale=0.09), R(heads=2, dim=128, vdim=64, rank=8), mlp=F(ff=96))],
             width=128, vocab=77),
        dict(layers=[P(L(heads=3, kv_heads=1, dim=33, vdim=65, scale=0.2), R(heads=5, dim=9, vdim=66, rank=3), mlp=E(experts=6, top=2, ff=21, shared=13)),
                     G(width=45, blocks=5, conv=3, mlp=E(experts=3, top=2, ff=16, shared=0))], width=66, vocab=50),
    ]
    for k, kw in enumerate(stacks):
        _run(make, tol, {"a": 380, "b": 5}, [[("a", 310), ("b", 2)], [("a", 60), ("b", 1)], [("a", 1), ("b", 2)]] + [[("a", 1)]] * 9, 20 + k,
             f"wider sizes {k}", cfg=_config(make, **kw))


def greedy_generation(make, tol, new=10):
    """batched_generate (the scheduler's own admission, chunking and retirement, greedy sampling on the device) against the
    oracle generating greedily; a position whose two best oracle logits are closer than the tolerance may differ."""
    from lmdeploy_b200.messages import GenerationConfig
    from lmdeploy_b200.turbomind.engine import batched_generate
    cfg = _config(make)
    w = _weights(make, cfg, seed=8)
    P = DC.prompts_for(cfg, {"a": 9, "b": 70, "c": 1})
    eng = make(cfg, w, blocks=4, max_batch=2, prefill_tokens=32)       # prompts longer than a step's token budget are chunked
    seqs = batched_generate(eng, [P[k] for k in "abc"], GenerationConfig(max_new_tokens=new, ignore_eos=True))
    assert eng.scheduler.alloc.num_free == 4 and sorted(eng.scheduler.slots) == [0, 1]
    for k, s in zip("abc", seqs):
        assert len(s.generated) == new and s.finish_reason == "length"
        toks = list(P[k]) + list(s.generated)
        logits = DC.oracle_logits(cfg, w, toks[:-1])
        for i, t in enumerate(s.generated):
            lg = logits[len(P[k]) - 1 + i]
            if int(lg.argmax()) != t:
                assert lg.max() - lg[t] <= 4 * tol * np.abs(lg).max(), f"{k}: token {i} is {t}, oracle {int(lg.argmax())}"


def score_scratch_in_row_chunks(make, tol):
    """The rows of a step pass through the attention in chunks when the scratch between its passes is bounded: chunks of 4
    rows here, cut inside sequences and between them."""
    cfg = _config(make)
    w = _weights(make, cfg, seed=36)
    P = DC.prompts_for(cfg, {"a": 93, "b": 21, "c": 3})
    eng = make(cfg, w)
    eng.model.window_scratch_bytes = 1
    got = DC.replay(eng, P, [[("a", 50), ("b", 21), ("c", 2)], [("a", 43), ("c", 1)]])
    for k in P:
        _check(got[k], DC.oracle_logits(cfg, w, P[k]), tol, f"row chunks {k}", make)


# ------------------------------------------------------------------------------------------------ one mechanism at a time
def marked_keys_and_growing_queries(make, tol, cuts=((230,), (61, 3, 35, 1, 1, 26, 1, 22, 45) + (1,) * 35)):
    """The attention side alone, with weights and inputs made so that single scores stand out.  Input channels 0..3 are markers: a row
    marked on channel c gets a KEY along dimension c and a QUERY along dimension (c + 1) % 4 of every head, so it gives every earlier
    key marked on channel c + 1 a large score and every other key nearly none: marked keys at a sequence's first token and at page
    borders (63, 64, 127, 128) must be found by queries more than a hundred keys later, in a prompt and decoded alone.  Channel 4 makes
    a row's query ask along dimension 4 with unit strength, and two keys (at 10 and 11) answer along it with scores that differ by less than one
    and opposite values: how their weights divide shows how far the query has grown.  Such queries stand on both sides of the places
    where the growth steps (98 | 99 and 198 | 199 with steps of 100).  The oracle itself is checked for showing the fault: without
    growth, with steps one position longer or shorter, or without one of the far keys its answer at those rows moves by a large part."""
    cfg = DC.config(layers=[DC.pair(DC.left(heads=4, kv_heads=2, dim=12, vdim=8, scale=0.5, q_temp=(1.5, 100)))])
    w = DC.random_tensors(cfg, seed=31)
    m = cfg["layers"][0]["mixer"]["left"]
    W, n, pre = cfg["width"], 230, "l0.mix.left."
    wq, wk = w[pre + "q"].view(4, 12, W), w[pre + "k"].view(2, 12, W)
    wq *= 0.02
    wk *= 0.02
    wq[:, :, :6] = 0.0
    wk[:, :, :6] = 0.0
    for c in range(4):
        wk[:, c, c] = 1.0
        wq[:, (c + 1) % 4, c] = 1.0
    wq[:, 4, 4] = 1.0                                     # channel 4: a gentle query along dimension 4
    wk[:, 4, 5] = 1.0                                     # channel 5: a key along dimension 4
    for k in ("q", "k"):
        w[pre + k] = w[pre + k].to(torch.bfloat16).float()
        w[pre + k + ".b"] = (0.02 * w[pre + k + ".b"]).to(torch.bfloat16).float()
    h = 0.2 * torch.randn(n, W, generator=torch.Generator().manual_seed(5))
    h[:, :7] = 0.0
    marks = [(0, 1, 8.0), (63, 2, 9.0), (64, 3, 7.0), (127, 1, -8.0), (128, 2, -9.0),           # keys
             (110, 0, 8.0), (120, 1, 8.0), (121, 2, 8.0), (160, 0, -8.0), (161, 1, -8.0), (228, 0, 8.0), (229, 2, 8.0)]    # 110, 228 -> 0;  120 -> 63;  121, 229 -> 64;
    for pos, ch, size in marks:                                                                 # 160 (negative) -> 127;  161 -> 128
        h[pos, ch] = size
    for pos in (98, 99, 198, 199, 100, 200):
        h[pos, 4] = 2.0
    h[10, 5], h[11, 5] = 14.0, 13.25
    for pos, tag in ((0, 20.0), (63, -20.0), (64, 20.0), (127, -20.0), (128, 20.0), (10, 20.0), (11, -20.0)):
        h[pos, 6] = tag                                    # reaches the values (and queries and keys fifty times weaker)
    h = h.to(torch.bfloat16).to(torch.float32)

    def oracle(mm, rows=h):
        return D.attention(rows.double(), _sub64(w, pre), mm, list(range(n)), D.new_attention_state(mm))

    want = oracle(m)
    size = lambda t: float(t.abs().max())
    for other, rows in ((dict(m, q_temp=None), (99, 199)), (dict(m, q_temp={"coef": 1.5, "every": 101}), (99,)),
                        (dict(m, q_temp={"coef": 1.5, "every": 99}), (98,)), (dict(m, q_temp={"coef": 1.0, "every": 100}), (99, 199, 200))):
        moved = oracle(other)
        for r in rows:
            assert size(moved[r] - want[r]) > 0.04 * size(want[r]), f"the oracle does not show {other['q_temp']} at row {r}: {size(moved[r] - want[r]) / size(want[r])}"
    for key, row in ((0, 110), (0, 228), (63, 120), (64, 121), (64, 229), (127, 160), (128, 161)):
        gone = h.clone()
        gone[key] = 0.0
        assert size(oracle(m, gone)[row] - want[row]) > 0.3 * size(want[row]), f"the oracle does not show key {key} at row {row}"
    for cut in cuts:
        eng = make(cfg, w)

        def run(model, lo, hi, c):
            L = model.spec.layers[0].mixer.left
            cols = (L.heads + L.kv_heads) * L.dim + L.kv_heads * L.vdim
            proj = model._linear(h[lo:hi].to(model.device, model.T).contiguous(), model.w["l0.in"])
            y = model.window_mixer(0, None, c, m=L, p="l0.left.", proj=proj[:, :cols])
            return torch.mm(y.float(), model.w["l0.left.o"].float().t())

        got = _in_portions(eng, n, cut, [2, 0, 1, 3], run)
        _close(got, want, tol, f"marked keys, portions {cut[:3]}...")


def gated_linear_attention_in_portions(make, tol):
    """The linear side alone over 300 rows: channels that remember hundreds of rows and channels that forget at once, a key and value
    twenty times the others' at row 3 that a slow state still holds at the end, as one prompt, in portions of one to three rows and
    token by token.  The oracle is checked for showing a lost state and a missing tau.  (The large row's own
    output is compared apart: it would hide the others' differences.)"""
    cfg = DC.config(layers=[DC.pair(r=DC.right(heads=3, dim=40, vdim=21, rank=4, tau=6.0))])
    w = DC.random_tensors(cfg, seed=32)
    pre = "l0.mix.right."
    w[pre + "a2.b"] = torch.linspace(-7.0, 9.0, 120).to(torch.bfloat16).float()             # decays from about 0.3 to 0.99998 per row
    m, n, W, eps = cfg["layers"][0]["mixer"]["right"], 300, cfg["width"], cfg["norm"]["eps"]
    h = torch.randn(n, W, generator=torch.Generator().manual_seed(6))
    h[3] *= 20.0
    h = h.to(torch.bfloat16).float()
    p64 = _sub64(w, pre)
    want = D.gated_linear_attention(h.double(), p64, m, eps, D.new_linear_state(m))
    size = lambda t: float(t.abs().max())
    half = torch.cat([want[:150], D.gated_linear_attention(h[150:].double(), p64, m, eps, D.new_linear_state(m))])
    assert size(half[-1] - want[-1]) > 0.3 * size(want[-1]), size(half[-1] - want[-1]) / size(want[-1])
    assert size(D.gated_linear_attention(h.double(), p64, dict(m, tau=1.0), eps, D.new_linear_state(m))[200:] - want[200:]) > 0.3 * size(want[200:])
    for cut in ((300,), (2, 1, 3, 1, 1, 60, 2, 5, 130, 64) + (1,) * 31):
        eng = make(cfg, w)

        def run(model, lo, hi, c):
            L = model.spec.layers[0].mixer.left
            cols = (L.heads + L.kv_heads) * L.dim + L.kv_heads * L.vdim
            proj = model._linear(h[lo:hi].to(model.device, model.T).contiguous(), model.w["l0.in"])
            y = model.gated_linear_mixer(0, proj[:, cols:], c, m=model.spec.layers[0].mixer.right, p="l0.right.")
            return torch.mm(y.float(), model.w["l0.right.o"].float().t())

        got = _in_portions(eng, n, cut, [0], run)
        rest = [t for t in range(n) if t != 3]
        _close(got[rest], want[rest], tol, f"gated linear attention, portions {cut[:3]}...")
        _close(got[3], want[3], tol, f"gated linear attention, row 3, portions {cut[:3]}...")


def rglru_in_portions(make, tol):
    """The real-gated recurrence alone over 300 rows with 4 and with 6 taps: channels that remember hundreds of rows and channels that
    forget at once, a row twenty times the others' early on, as one prompt (several tiles of the scan), in portions shorter than the
    convolution, ending inside and at the edges of a tile, and token by token; the first token has no special case (its input is scaled
    by sqrt(1 - a^2) like any other)."""
    for taps in (4, 6):
        cfg = DC.config(layers=[DC.rglru(width=42, blocks=3, conv=taps)])
        w = DC.random_tensors(cfg, seed=33 + taps)
        w["l0.mix.lam"] = torch.linspace(-10.0, 1.5, 42).to(torch.bfloat16).float()
        m, n, W = cfg["layers"][0]["mixer"], 300, cfg["width"]
        h = torch.randn(n, W, generator=torch.Generator().manual_seed(7))
        h[2] *= 20.0
        h = h.to(torch.bfloat16).float()
        p64 = _sub64(w, "l0.mix.")
        want = D.rglru(h.double(), p64, m, D.new_rglru_state(m))
        half = D.rglru(h[150:].double(), p64, m, D.new_rglru_state(m))
        assert float((half[0] - want[150]).abs().max()) > 0.1 * float(want[150].abs().max())
        for cut in ((300,), (2, 1, 3, 1, 1, 56, 2, 5, 128, 64) + (1,) * 37, (128, 128, 44), (127, 2, 129, 42)):
            eng = make(cfg, w)

            def run(model, lo, hi, c):
                y = model.rglru_mixer(0, h[lo:hi].to(model.device, model.T).contiguous(), c)
                return torch.mm(y.float(), model.w["l0.o"].float().t())

            got = _in_portions(eng, n, cut, [0], run)
            large = [t for t in range(n) if 2 <= t < 2 + taps]                 # the rows whose convolution sees it
            rest = [t for t in range(n) if t not in large]
            _close(got[rest], want[rest], tol, f"rglru, {taps} taps, portions {cut[:3]}...")
            _close(got[large], want[large], tol, f"rglru, {taps} taps, rows of the large input, portions {cut[:3]}...")


def router_alone(make, tol):
    """The router on inputs made so that its rules show: the input is one-hot, so a row's logits are a column of the router matrix plus
    the bias.  Row 0: the bias changes the choice AND the weights.  Row 1: the weights are the softmax over the two chosen logits only.
    Row 2: logits of hundreds.  Row 3: a tie goes to the lower index.  Then random rows against the oracle, few (expert-major
    kernels) and many (grouped GEMMs), the shared expert beside them."""
    cfg = DC.config(layers=[DC.pair(mlp=DC.moe(experts=6, top=2, ff=24, shared=20))], width=48)
    w = DC.random_tensors(cfg, seed=34)
    W = cfg["width"]
    rows = [[0.0, 2.0, 1.0, -1.0, 0.5, 1.5],               # + bias: expert 3 wins with 3
            [1.0, 0.5, -2.0, -9.0, 0.75, 0.0],             # 0 and 4: softmax(1, 0.75) over the two, not over all six
            [300.0, -300.0, 298.0, -500.0, 0.0, 100.0],    # 0 and 2
            [0.5, 1.25, 1.25, -9.0, 1.25, 0.0]]            # 1 and 2, not 4
    router = 0.3 * torch.randn(6, W, generator=torch.Generator().manual_seed(3))
    for r, logits in enumerate(rows):
        router[:, r] = torch.tensor(logits)
    w["l0.mlp.router"] = router.to(torch.bfloat16).float()
    w["l0.mlp.router.b"] = torch.tensor([0.0, 0.0, 0.0, 4.0, 0.0, 0.0])
    model = make(cfg, w).model
    f, p64 = cfg["layers"][0]["mlp"], _sub64(w, "l0.mlp.")

    def routed(h):
        t = h.to(model.device, model.T).contiguous()
        out = model.routed_experts(0, h.to(model.device).contiguous(), t, h.shape[0]).sum(1)
        out = out + model.gated_mlp(t, model.w["l0.shared.up"], model.w["l0.shared.down"]).float()
        ids, wts = model.last_routing
        return out.cpu(), ids.cpu().tolist(), wts.cpu()

    special = torch.eye(4, W)
    _, ids, wts = routed(special)
    assert ids == [[3, 1], [0, 4], [0, 2], [1, 2]], ids
    _close(wts, torch.softmax(torch.tensor([[3.0, 2.0], [1.0, 0.75], [300.0, 298.0], [1.25, 1.25]], dtype=torch.float64), -1), 1e-5, "weights")
    for n in (7, 200):
        h = torch.randn(n, W, generator=torch.Generator().manual_seed(8)).to(torch.bfloat16).float()
        got, _, _ = routed(h)
        _close(got, D.routed_ff(h.double(), p64, f), tol, f"experts on {n} rows")


def gated_feed_forward_alone(make, tol):
    """The dense feed-forward alone, inner sizes that are and are not multiples of four."""
    for ff in (40, 37):
        cfg = DC.config(layers=[DC.rglru(mlp=DC.dense(ff=ff))])
        w = DC.random_tensors(cfg, seed=35)
        h = 2.0 * torch.randn(50, cfg["width"], generator=torch.Generator().manual_seed(9)).to(torch.bfloat16).float()
        model = make(cfg, w).model
        got = model.dense_mlp(0, h.to(model.device, model.T).contiguous())
        _close(got.float().cpu(), D.gated_ff(h.double(), _sub64(w, "l0.mlp.")), tol, f"dense feed-forward of {ff}")


def norms_on_both_ends_and_residual(make, tol):
    """The stream takes in a sublayer's normed output -- half the sum of two normed sides, one row, or the experts' float parts beside
    a shared row -- and the next norm reads it; outputs far larger and far smaller than the stream; widths for vector and for scalar
    accesses; with nothing to take in the stream is only normed."""
    from lmdeploy_b200 import _hybrid_lib as H
    for W in (48, 33):
        cfg = DC.config(layers=[DC.pair(mlp=DC.moe())], width=W)
        w = DC.random_tensors(cfg, seed=37)
        model = make(cfg, w).model
        n, eps, dev, T = 37, cfg["norm"]["eps"], model.device, model.T
        g = torch.Generator().manual_seed(9)
        rnd = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).float()
        x0, lf, rt, row, ff = rnd(n, W), 4.0 * rnd(n, W), 0.25 * rnd(n, W), 16.0 * rnd(n, W), rnd(n, 3, W)          # powers of two keep the values in bfloat16
        wt = {k: w["l0." + k].double() for k in ("mix.left.out", "mix.right.out", "norm1b", "norm2b", "norm2")}
        sides = 0.5 * (D.unit_rms(lf.double(), eps) * wt["mix.left.out"] + D.unit_rms(rt.double(), eps) * wt["mix.right.out"])
        cases = {"sides": (sides, "norm1b"), "row": (row.double(), "norm2b"), "parts": (row.double() + ff.double().sum(1), "norm2b"), "none": (None, None)}
        for case, (y, post) in cases.items():
            xs = x0.double() if y is None else x0.double() + D.unit_rms(y, eps) * wt[post]
            x = x0.clone().to(dev).contiguous()
            d = {k: t.to(dev, torch.float32 if k == "ff" else T).contiguous() for k, t in (("l", lf), ("r", rt), ("m", row), ("ff", ff))}
            h, hf = torch.empty(n, W, dtype=T, device=dev), torch.empty(n, W, dtype=torch.float32, device=dev)
            at = lambda key, use: d[key].data_ptr() if use else None
            mw = model.w
            H.check(model.lib.b200h_normed_residual_norm(
                x.data_ptr(), at("l", case == "sides"), at("r", case == "sides"), mw["l0.left.out"].data_ptr(), mw["l0.right.out"].data_ptr(), 0.5,
                at("m", case in ("row", "parts")), at("ff", case == "parts"), 3 if case == "parts" else 0,
                None if post is None else mw["l0." + post].data_ptr(), mw["l0.norm2"].data_ptr(), n, W, eps, h.data_ptr(), hf.data_ptr(), model.dt,
                model._stream()))
            _close(x.cpu(), xs, 2e-6, f"{case}, width {W}: stream after the add")
            _close(hf.cpu(), D.unit_rms(xs, eps) * wt["norm2"], 2e-6, f"{case}, width {W}: norm as float")
            _close(h.float().cpu(), D.unit_rms(xs, eps) * wt["norm2"], tol, f"{case}, width {W}: norm")


def decays_alone(make, tol):
    """sigmoid(z)^(1/tau) for z from far below to far above zero (a decay of nearly one keeps its distance from one), many rows and
    few, odd and even channel counts."""
    from lmdeploy_b200 import _hybrid_lib as H
    cfg = DC.config()
    model = make(cfg, DC.random_tensors(cfg)).model
    dev, T = model.device, model.T
    g = torch.Generator().manual_seed(4)
    for n, channels, rank, tau in ((3, 33, 5, 16.0), (700, 2048, 9, 1.0), (2500, 257, 64, 3.5)):
        low = torch.randn(n, rank + 3, generator=g).to(torch.bfloat16).float()
        a = torch.randn(channels, rank, generator=g).to(torch.bfloat16).float() / 4
        b = torch.linspace(-30.0, 12.0, channels)
        z = low[:, :rank].double() @ a.double().T + b.double()
        want = D.sigmoid(z).pow(1.0 / tau)
        out = torch.empty(n, channels, dtype=torch.float32, device=dev)
        lo, aw, bw = low.to(dev, T).contiguous(), a.t().to(dev, T).contiguous(), b.to(dev)
        H.check(model.lib.b200h_low_rank_decay(lo.data_ptr(), rank + 3, aw.data_ptr(), bw.data_ptr(), n, channels, rank, tau, out.data_ptr(), model.dt,
                                               model._stream()))
        _close(out.cpu(), want, 2e-6, f"decays {n} x {channels}")


def real_gates_keep_their_distance_from_one(make, tol):
    """The scan alone with decays within 1e-6 of one: 1 - a^2 keeps its relative accuracy (a square root of it multiplies the input), and
    the state after many rows is the sum of the inputs so weighted."""
    from lmdeploy_b200 import _hybrid_lib as H
    cfg = DC.config(layers=[DC.rglru(width=40, blocks=4, conv=2)])
    eng = make(cfg, DC.random_tensors(cfg))
    model = eng.model
    dev, T, n, R = model.device, model.T, 200, 40
    g = torch.Generator().manual_seed(5)
    z = torch.randn(4, n, 20, generator=g)
    u, xy = torch.rand(n, R, generator=g).to(torch.bfloat16).float(), torch.randn(n, 2 * R, generator=g).to(torch.bfloat16).float()
    lam = torch.linspace(-16.0, -2.0, R)
    r, i = (D.sigmoid(z.double().view(4, n, 2, 10)[:, :, k].permute(1, 0, 2).reshape(n, R)) for k in range(2))
    la = -8.0 * r * D.softplus(lam.double())
    S, want = torch.zeros(R, dtype=torch.float64), torch.zeros(n, R, dtype=torch.float64)
    for t in range(n):
        S = torch.exp(la[t]) * S + torch.sqrt(-torch.expm1(2 * la[t])) * i[t] * u[t].double()
        want[t] = S * D.gelu_tanh(xy[t, :R].double())
    eng.state.reset(0)
    from fogizen_scenarios import _step_arrays
    c = _step_arrays(eng, 0, n, [0, 1, 2, 3], slot=0)
    p, zd, ud, lm = xy.to(dev, T).contiguous(), z.to(dev).contiguous(), u.to(dev, T).contiguous(), lam.to(dev)
    out = torch.empty(n, R, dtype=T, device=dev)
    a = H.RgLruArgs()
    a.n, a.batch, a.width, a.blocks, a.taps, a.rate = n, 1, R, 4, 2, 8.0
    a.y, a.x, a.ld, a.u, a.z, a.lam, a.out = p.data_ptr(), p.data_ptr() + p.element_size() * R, 2 * R, ud.data_ptr(), zd.data_ptr(), lm.data_ptr(), out.data_ptr()
    a.conv = model.w["l0.conv"].data_ptr()
    a.conv_state, a.state, a.slot_stride = c.state.ptr(model.conv_off[0]), c.state.ptr(model.mix_off[0]), c.state.storage.stride(0)
    a.tok_seq, a.cu_q, a.seq_slot, a.dtype, a.stream = c.tok_seq.data_ptr(), c.cu_q.data_ptr(), c.seq_slot.data_ptr(), model.dt, model._stream()
    H.check(model.lib.b200h_real_gated_scan(C.byref(a)))
    got = out.float().cpu().double()
    scale = want.abs().amax(0).clamp_min(1e-30)                                  # channel by channel: the slow channels are small
    assert float(((got - want).abs() / scale).max()) <= max(tol, 1e-5)
    state = eng.state.storage[0, model.mix_off[0]:model.mix_off[0] + R].cpu().double()
    assert float(((state - S).abs() / S.abs()).max()) <= 1e-5


MECHANISMS = [decays_alone, real_gates_keep_their_distance_from_one, norms_on_both_ends_and_residual, gated_feed_forward_alone, router_alone,
              gated_linear_attention_in_portions, rglru_in_portions, marked_keys_and_growing_queries]
ENGINE = [score_scratch_in_row_chunks, whole_prompt, layer_by_layer, prefill_then_decode, token_by_token, portions, unequal_batch,
          left_out_and_resumed, reuse_of_pages_and_slots, other_sizes, wider_sizes, greedy_generation]
ALL = MECHANISMS + ENGINE

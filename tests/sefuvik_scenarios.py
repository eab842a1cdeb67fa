"""Scenarios every engine serving a Sefuvik decoder must pass, whatever runs its operators: `make(cfg, tensors, **kw)` builds
the engine (sefuvik_cases.build_engine with a device, dtype and library chosen by the caller), `tol` bounds
hybrid_cases.rel_error against the float64 oracle.  Run on the CPU through the numpy stand-in (tests/test_sefuvik_cpu.py: host
logic -- pages, slots, row addressing, scheduling, state offsets) and on a GPU through the CUDA kernels (tests/test_sefuvik_gpu.py)."""
import ctypes as C

import numpy as np
import torch

import sefuvik_cases as DC
from fogizen_scenarios import _close, _in_portions, _step_arrays, _sub64
from oracle import sefuvik as D


def _size(t):
    return float(t.abs().max())


def _check(got, want, tol, what, make=None):
    """Every position within tol; for an engine whose projections are rounded (make.rounded) one position in fifty may reach 2.5 tol: a
    unit norm over a head's few channels now and then divides by a small root mean square, which multiplies the rounding of what it norms
    at that lone position.  (A fault of a page, a slot or a state moves all positions after it.)"""
    err = DC.rel_error(got, want)
    lone = max(1, len(err) // 50) if getattr(make, "rounded", False) else 0
    worst = np.sort(err)[::-1]
    assert worst[0] <= (2.5 * tol if lone else tol), f"{what}: relative error {err.max():.3g} at position {int(err.argmax())} (bound {tol})"
    assert len(err) <= lone or worst[lone] <= tol, f"{what}: relative error {worst[lone]:.3g} at {lone + 1} positions (bound {tol})"


def _weights(make, cfg, seed=0):
    """DC.random_tensors for an engine built by `make`.  Where a head of a recurrence has seen one token, its unit norm leaves the SIGN of
    q.k times a unit value: with q.k near zero rounding decides it.  Engines whose projections are rounded (make.rounded) get keys (and
    key convolutions) that lie along the queries; float32 engines take the weights as they come."""
    w = DC.random_tensors(cfg, seed=seed)
    if getattr(make, "rounded", False):
        for i, e in enumerate(cfg["layers"]):
            p = {"retention": f"l{i}.mix.", "parallel": f"l{i}.mix.right."}.get(e["type"])
            for name in ("k", "k.conv"):
                if p and p + name in w:
                    w[p + name] = (w[p + name.replace("k", "q", 1)] + 0.25 * w[p + name]).to(torch.bfloat16).float()
    return w


def _run(make, tol, lengths, schedule, seed, what, cfg=None, **kw):
    """A schedule against the oracle on every request's whole token list -> the engine."""
    cfg = cfg or DC.config()
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
    """The sum of the streams after every layer against the oracle's."""
    cfg = DC.config()
    w = _weights(make, cfg, seed=2)
    P = DC.prompts_for(cfg, {"a": 80})
    eng = make(cfg, w)
    eng.layer_trace = []
    got = DC.replay(eng, P, [[("a", 80)]])
    want = []
    logits = DC.oracle_logits(cfg, w, P["a"], trace=want)
    assert len(eng.layer_trace) == len(want) == 6
    for r, (g, x) in enumerate(zip(eng.layer_trace, want)):
        err = _size(g.double().cpu() - x) / _size(x)
        assert err <= tol, f"streams after layer {r}: {err:.3g} of their largest value (bound {tol})"
    _check(got["a"], logits, tol, "logits of a traced step", make)


def prefill_then_decode(make, tol, n=200, tail=120):
    """Most of a prompt in one step, the rest token by token: decoded tokens cross page borders (127 -> 128, 191 -> 192), the window
    passes over them, chunks end among them; the recurrences are carried over more than a hundred single-token steps."""
    _run(make, tol, {"a": n}, [[("a", n - tail)]] + [[("a", 1)]] * tail, 3, "prefill then decode")


def token_by_token(make, tol, n=110):
    """Every token alone from the first: zero states, zeros before the convolutions, a lone key; the first window and the first chunks
    fill and pass."""
    _run(make, tol, {"a": n}, [[("a", 1)]] * n, 4, "token by token")


def portions(make, tol):
    """Portions of several sizes down to one and two tokens (shorter than the convolutions), cut inside pages and at their borders, inside
    windows and chunks (41, 70) and at their edges, around multiples of eight rows."""
    cuts = [2, 3, 1, 2, 29, 4, 9, 14, 2, 1, 3, 30, 28, 2, 64, 5, 8, 16, 2, 113, 7, 2]
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
    """Sizes that a given model may make equal or 1: one layer of every kind alone; one stream, two, eight; one head; as many key/value
    heads as heads; value heads wider and narrower than key heads everywhere; windows of one key, no kept tokens, more kept tokens than the
    window, no mask; chunks of one position, no chunks; all or no dimensions turning; 1 tap and 7 taps; low-rank sizes of 1 and unequal
    ones; states that are not 16-byte aligned and wider than 128 channels; odd widths; a difference factor of 0 and of nearly 1; scales of
    0 and below it; no feed-forward."""
    A, R, P, L, G, F = DC.attention, DC.retention, DC.pair, DC.left, DC.right, DC.dense
    stacks = [
        dict(layers=[A(heads=1, kv_heads=1, dim=4, vdim=4, size=1, keep_first=0, diff=0.0)], width=16, vocab=9, streams=1),
        dict(layers=[R(heads=1, dim=4, vdim=6, decay=(0.75,), dims=4)], width=16, vocab=9, streams=2),
        dict(layers=[P(L(heads=1, kv_heads=1, dim=4, vdim=4, size=1, dims=4), G(heads=1, kv_heads=1, dim=4, vdim=4, conv=1, a1_rank=1, g1_rank=2),
                       left_scale=-0.5, right_scale=1.0)], width=16, vocab=9, streams=8),
        dict(layers=[A(heads=5, kv_heads=5, dim=3, vdim=7, size=9, keep_first=20, diff=0.9, mlp=F(ff=7)),
                     P(L(heads=6, kv_heads=2, dim=8, vdim=5, size=0, dims=2), G(heads=6, kv_heads=1, dim=40, vdim=3, conv=7, a1_rank=9, g1_rank=1),
                       left_scale=1.0, right_scale=0.0, mlp=F(ff=9)),
                     R(heads=4, dim=5, vdim=3, decay=(1.0, 0.9, 0.99, 0.2), dims=2)], width=24, vocab=33, streams=5),
        dict(layers=[R(heads=1, dim=130, vdim=34, decay=(0.97,), dims=64, mlp=F(ff=9)), A(heads=2, kv_heads=1, dim=9, vdim=5, size=0, keep_first=0),
                     P(L(heads=2, kv_heads=2, dim=5, vdim=3, size=17, dims=4), G(heads=2, kv_heads=2, dim=132, vdim=17, conv=3, a1_rank=3, g1_rank=5),
                       left_scale=0.0, right_scale=1.5, mlp=F(ff=11))], width=33, vocab=20, streams=3),
    ]
    for k, kw in enumerate(stacks):
        _run(make, tol, {"a": 131, "b": 4}, [[("a", 3)], [("a", 62), ("b", 2)], [("a", 1), ("b", 1)], [("a", 1)], [("a", 62), ("b", 1)], [("a", 1)],
                                             [("a", 1)]], 10 + k, f"sizes {k}", cfg=DC.config(**kw))


def wider_sizes(make, tol):
    """Sizes of the order of a real layer's heads: 16 query heads on 2 key/value heads, head dimensions of 64 and 128 (16-byte key reads) and
    an odd one (scalar reads), wide value heads, recurrent heads of 64, 128 and 256 channels, feed-forward widths that are and are not
    multiples of eight, prompts long enough for several rows per block, key ranges, kept tokens far behind a window."""
    A, R, P, L, G, F = DC.attention, DC.retention, DC.pair, DC.left, DC.right, DC.dense
    stacks = [
        dict(layers=[A(heads=16, kv_heads=2, dim=64, vdim=64, scale=0.125, size=100, keep_first=5, mlp=F(ff=160)),
                     R(heads=2, dim=256, vdim=64, decay=(0.99, 0.9), dims=256),
                     P(L(heads=4, kv_heads=4, dim=128, vdim=32, scale=0.09, size=150, dims=64), G(heads=4, kv_heads=2, dim=64, vdim=64, a1_rank=16, g1_rank=8),
                       mlp=F(ff=96)),
                     R(heads=3, dim=64, vdim=48, decay=(0.99, 0.9, 0.5), dims=64, mlp=F(ff=45))], width=128, vocab=77, streams=4),
        dict(layers=[P(L(heads=3, kv_heads=1, dim=33, vdim=65, scale=0.2, size=130, dims=12), G(heads=5, kv_heads=5, dim=128, vdim=66, conv=4, a1_rank=7, g1_rank=9)),
                     A(heads=6, kv_heads=3, dim=17, vdim=33, scale=0.25, size=77, keep_first=9, mlp=F(ff=21))], width=66, vocab=50, streams=2),
    ]
    for k, kw in enumerate(stacks):
        _run(make, tol, {"a": 380, "b": 5}, [[("a", 310), ("b", 2)], [("a", 60), ("b", 1)], [("a", 1), ("b", 2)]] + [[("a", 1)]] * 9, 20 + k,
             f"wider sizes {k}", cfg=DC.config(**kw))


def greedy_generation(make, tol, new=10):
    """batched_generate (the scheduler's own admission, chunking and retirement, greedy sampling on the device) against the
    oracle generating greedily; a position whose two best oracle logits are closer than the tolerance may differ."""
    from lmdeploy_b200.messages import GenerationConfig
    from lmdeploy_b200.turbomind.engine import batched_generate
    cfg = DC.config()
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
    cfg = DC.config()
    w = _weights(make, cfg, seed=36)
    P = DC.prompts_for(cfg, {"a": 93, "b": 21, "c": 3})
    eng = make(cfg, w)
    eng.model.window_scratch_bytes = 1
    got = DC.replay(eng, P, [[("a", 50), ("b", 21), ("c", 2)], [("a", 43), ("c", 1)]])
    for k in P:
        _check(got[k], DC.oracle_logits(cfg, w, P[k]), tol, f"row chunks {k}", make)


# ------------------------------------------------------------------------------------------------ one mechanism at a time
def _left_alone(model, h):
    """The attention side of layer 0's paired mixer, projected and scaled as the mixer's sum takes it."""
    m = model.spec.layers[0].mixer
    proj = model._linear(h.to(model.device, model.T).contiguous(), model.w["l0.in"])
    cols = m.left.heads * m.left.vdim

    def run(c):
        y = model.window_mixer(0, None, c, m=m.left, p="l0.left.", proj=proj, scale=m.scales[0])
        return torch.mm(y.float(), model.w["l0.o"][:, :cols].float().t())
    return run


def _right_alone(model, h):
    m = model.spec.layers[0].mixer
    proj = model._linear(h.to(model.device, model.T).contiguous(), model.w["l0.in"])
    lo, cols = m.left.heads * m.left.vdim, m.right.heads * m.right.vdim

    def run(c):
        y = torch.empty(c.n, cols, dtype=model.T, device=model.device)
        model.gated_delta_mixer(0, proj, c, 0, m.right, "l0.right.", model.w["l0.cols"], y)
        return torch.mm(y.float(), model.w["l0.o"][:, lo:lo + cols].float().t())
    return run


CUTS = ((230,), (61, 3, 35, 1, 1, 26, 1, 22, 45) + (1,) * 35)


def marked_keys_windows_and_first_tokens(make, tol):
    """Differential attention alone, with weights and inputs made so that single scores stand out.  Input channels 0..3 are markers: a row
    marked on channel c gets a KEY along dimension c of both maps, a QUERY along dimension (c + 1) % 4 of map 1 and along (c + 2) % 4 of map
    2; every other score is nearly zero.  A window of 50 keys keeps the first 3.  Marked keys sit among the kept tokens (0, 2), right
    behind them (3), at page borders (63, 64, 127, 128) and elsewhere; the queries come from just inside and just outside the windows of those
    keys, and from far away for the kept ones, in a prompt and decoded alone.  The oracle is checked for showing the fault: with a window
    one longer or shorter, one kept token more or fewer or none, maps exchanged, another factor, its answer at those rows moves by a
    large part."""
    cfg = DC.config(layers=[DC.attention(heads=4, kv_heads=2, dim=12, vdim=8, scale=0.5, size=50, keep_first=3, diff=0.4)])
    w = DC.random_tensors(cfg, seed=31)
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    W, n, pre = cfg["width"], 230, "l0.mix."
    wq, wk = w[pre + "q"].view(4, 2, 12, W), w[pre + "k"].view(2, 2, 12, W)
    for t in (wq, wk):
        t *= 0.02
        t[..., :7] = 0.0
    for c in range(4):
        wk[:, :, c, c] = 1.0
        wq[:, 0, (c + 1) % 4, c] = 1.0
        wq[:, 1, (c + 2) % 4, c] = 1.0
    for k in ("q", "k"):
        w[pre + k] = w[pre + k].to(torch.bfloat16).float()
        w[pre + k + ".b"] = (0.02 * w[pre + k + ".b"]).to(torch.bfloat16).float()
    h = 0.2 * torch.randn(n, W, generator=torch.Generator().manual_seed(5))
    h[:, :8] = 0.0
    # keys: 0 (kept) on 1, 2 (kept) on 2, 3 (not kept) on 3; 63, 64, 127, 128 at page borders
    marks = [(0, 1, 8.0), (2, 2, 9.0), (3, 3, 9.0), (63, 3, 9.0), (64, 2, -8.0), (127, 3, 9.0), (128, 0, 10.0),
             (52, 2, 8.0), (53, 2, 8.0),                   # map 1 -> key 3: at 52 just inside, at 53 just outside
             (112, 2, 8.0), (113, 2, 8.0),                 # map 1 -> key 63 likewise
             (110, 0, 8.0), (111, 0, 8.0),                 # map 1 -> key 0, map 2 -> key 2: kept, far away
             (176, 2, 8.0), (177, 2, 8.0),                 # map 1 -> key 127
             (178, 3, 9.0), (179, 3, 9.0),                 # map 1 -> key 128: at 178 already outside
             (114, 1, -8.0),                               # map 1 -> key 64 is outside (114 - 64 = 50): key 2 answers
             (228, 0, 8.0), (229, 1, 8.0)]                 # kept keys 0 and 2 across three pages
    for pos, ch, size in marks:
        h[pos, ch] = size
    for pos, tag in ((0, 20.0), (2, -20.0), (3, 20.0), (63, -20.0), (64, 20.0), (127, 20.0), (128, -20.0)):
        h[pos, 6], h[pos, 7] = tag, -0.5 * tag             # reach the values
    h = h.to(torch.bfloat16).to(torch.float32)

    def oracle(mm, rows=h, p=None):
        return D.differential_attention(rows.double(), p or _sub64(w, pre), mm, eps, list(range(n)), D.new_differential_state(mm))

    want = oracle(m)
    mask = lambda size, keep: dict(m, mask={"size": size, "keep_first": keep})
    swapped = dict(_sub64(w, pre))
    for k in ("q", "k"):
        swapped[k] = swapped[k].view(-1, 2, 12, W).flip(1).reshape(-1, W)
    cases = [(oracle(mask(51, 3)), (53, 113, 177)), (oracle(mask(49, 3)), (52, 112, 176)), (oracle(mask(50, 2)), (110, 111, 228, 229)),
             (oracle(mask(50, 4)), (53, 113)), (oracle(mask(50, 0)), (110, 228, 229)), (oracle(m, p=swapped), (110, 112, 228)),
             (oracle(dict(m, diff=0.1)), (110, 228))]
    for k, (moved, rows) in enumerate(cases):
        for r in rows:
            assert _size(moved[r] - want[r]) > 0.15 * _size(want[r]), f"the oracle does not show fault {k} at row {r}: {_size(moved[r] - want[r]) / _size(want[r])}"
    for key, row in ((0, 110), (2, 228), (3, 52), (63, 112), (127, 176), (128, 177)):
        gone = h.clone()
        gone[key] = 0.0
        if (key, row) != (128, 177):
            assert _size(oracle(m, gone)[row] - want[row]) > 0.15 * _size(want[row]), f"the oracle does not show key {key} at row {row}"
    for cut in CUTS:
        eng = make(cfg, w)

        def run(model, lo, hi, c):
            y = model.window_mixer(0, h[lo:hi].to(model.device, model.T).contiguous(), c)
            return torch.mm(y.float(), model.w["l0.o"].float().t())

        _close(_in_portions(eng, n, cut, [2, 0, 1, 3], run), want, tol, f"marked keys, portions {cut[:3]}...")


def marked_keys_chunks_and_sinks(make, tol):
    """The chunked side alone.  Heads of 12 dimensions of which the first 4 turn; chunks of 100 positions.  Markers as above (one map) along
    the dimensions that do not turn.  Marked keys sit at a sequence's first token, at page borders (63, 64, 127, 128) and on both sides of the chunk
    edges (99 | 100, 199 | 200); the queries that must find them -- or must NOT, by one position -- come up to 99 keys later, in a prompt
    and decoded alone.  A row early in its chunk shares its weights with the sink.  The oracle is checked for showing chunks one position
    longer or shorter, no chunks, no sink, another rotation."""
    cfg = DC.config(layers=[DC.pair(DC.left(heads=4, kv_heads=2, dim=12, vdim=8, size=100, dims=4, base=30.0, scale=0.5), left_scale=0.7)])
    w = DC.random_tensors(cfg, seed=37)
    M = cfg["layers"][0]["mixer"]
    m, W, n, pre = M["left"], cfg["width"], 230, "l0.mix.left."
    wq, wk = w[pre + "q"].view(4, 12, W), w[pre + "k"].view(2, 12, W)
    for t in (wq, wk):
        t[:, :4] *= 1.5                                    # the turning part keeps ordinary scores
        t[:, 4:] *= 0.02
        t[..., :8] = 0.0
    for c in range(4):
        wk[:, 4 + c, c] = 1.0
        wq[:, 4 + (c + 1) % 4, c] = 1.0
    for k in ("q", "k"):
        w[pre + k] = w[pre + k].to(torch.bfloat16).float()
    w[pre + "sink"] = torch.tensor([0.0, 3.0, -1.0, 4.0])
    h = 0.3 * torch.randn(n, W, generator=torch.Generator().manual_seed(5))
    h[:, :8] = 0.0
    marks = [(0, 1, 8.0), (63, 2, 9.0), (64, 3, 7.0), (99, 1, -8.0),                           # chunk 0: keys
             (90, 0, 8.0), (91, 1, 8.0), (92, 2, 8.0),                                         #   90 -> 0;  91 -> 63;  92 -> 64
             (100, 1, 9.0), (127, 2, -9.0), (128, 3, -9.0),                                    # chunk 1: keys
             (150, 0, 8.0), (151, 1, 8.0), (152, 2, -8.0), (199, 0, 8.0),                      #   150, 199 -> 100, NOT 99 or 0;  151 -> 127;  152 -> 128
             (200, 0, 8.0), (201, 3, 8.0), (229, 3, 8.0)]                                      # chunk 2: 200 -> nothing (not 100);  201, 229 -> 200, NOT 199
    for pos, ch, size in marks:
        h[pos, ch] = size
    for pos, tag in ((0, 30.0), (63, -30.0), (64, 30.0), (99, 30.0), (100, -30.0), (127, 30.0), (128, -30.0), (199, 30.0), (200, -30.0)):
        h[pos, 6] = tag
    h = h.to(torch.bfloat16).to(torch.float32)

    def oracle(mm, p=None):
        return 0.7 * D.chunked_attention(h.double(), p or _sub64(w, pre), mm, list(range(n)), D.new_chunked_state(mm))

    want = oracle(m)
    none = dict(_sub64(w, pre), sink=torch.full((4,), -1e4, dtype=torch.float64))
    cases = [(oracle(dict(m, mask=None)), (200, 201)), (oracle(dict(m, mask={"size": 101})), (199, 201)), (oracle(dict(m, mask={"size": 99})), (199, 229)),
             (oracle(m, none), (1, 100, 200, 202)), (oracle(dict(m, rot={"dims": 4, "base": 31.0})), (120, 190)), (oracle(dict(m, rot={"dims": 2, "base": 30.0})), (50, 120))]
    for k, (moved, rows) in enumerate(cases):
        for r in rows:
            assert _size(moved[r] - want[r]) > (0.004 if k == 4 else 0.1) * _size(want[r]), f"the oracle does not show fault {k} at row {r}: {_size(moved[r] - want[r]) / _size(want[r])}"
    for cut in CUTS:
        eng = make(cfg, w)
        _close(_in_portions(eng, n, cut, [2, 0, 1, 3], lambda model, lo, hi, c: _left_alone(model, h[lo:hi])(c)), want, tol, f"chunks and sinks, portions {cut[:3]}...")


def retention_in_portions(make, tol):
    """Retention alone over 300 rows: heads that forget at once, that remember hundreds of rows and that never forget; a key and value twenty
    times the others' at row 3 that slow states still hold at the end; as one prompt, in portions of one to three rows, around multiples of
    eight rows and token by token.  The oracle is checked for showing a lost state, another decay, no rotation and a rotation of neighbouring
    dimensions.  (The large row's own output is compared apart: it would hide the others' differences.)"""
    for kw in (dict(heads=4, dim=40, vdim=21, decay=(0.3, 0.99, 0.9990234375, 1.0), dims=32, base=300.0), dict(heads=2, dim=7, vdim=50, decay=(0.999, 0.9), dims=4, base=40.0)):
        cfg = DC.config(layers=[DC.retention(**kw)])
        w = DC.random_tensors(cfg, seed=32)
        if getattr(make, "rounded", False):
            w["l0.mix.k"] = (w["l0.mix.q"] + 0.25 * w["l0.mix.k"]).to(torch.bfloat16).float()
        m, n, W, eps = cfg["layers"][0]["mixer"], 300, cfg["width"], cfg["norm"]["eps"]
        h = torch.randn(n, W, generator=torch.Generator().manual_seed(6))
        h[3] *= 20.0
        h = h.to(torch.bfloat16).float()
        p64 = _sub64(w, "l0.mix.")
        want = D.retention(h.double(), p64, m, eps, list(range(n)), D.new_retention_state(m))
        half = torch.cat([want[:150], D.retention(h[150:].double(), p64, m, eps, list(range(150, n)), D.new_retention_state(m))])
        assert _size(half[-1] - want[-1]) > 0.1 * _size(want[-1]), _size(half[-1] - want[-1]) / _size(want[-1])
        for other in (dict(m, decay=[d * 0.998 for d in m["decay"]]), dict(m, rot={"dims": 0, "base": 1.0}), dict(m, rot=dict(m["rot"], dims=m["rot"]["dims"] - 2))):
            assert _size(D.retention(h.double(), p64, other, eps, list(range(n)), D.new_retention_state(m))[200:] - want[200:]) > 0.05 * _size(want[200:]), other
        for cut in ((300,), (2, 1, 3, 1, 1, 60, 2, 5, 130, 64) + (1,) * 31, (8, 16, 7, 9, 24, 236)):
            eng = make(cfg, w)

            def run(model, lo, hi, c):
                y = model.retention_mixer(0, h[lo:hi].to(model.device, model.T).contiguous(), c)
                return torch.mm(y.float(), model.w["l0.o"].float().t())

            got = _in_portions(eng, n, cut, [0], run)
            rest = [t for t in range(n) if t != 3]
            _close(got[rest], want[rest], tol, f"retention, portions {cut[:3]}...")
            _close(got[3], want[3], tol, f"retention, row 3, portions {cut[:3]}...")


def gated_delta_rule_in_portions(make, tol):
    """The gated delta rule alone over 300 rows with 4, 6 and 1 taps: channels that remember hundreds of rows and channels that forget at
    once, key/value heads shared by several heads, a row twenty times the others' early on; as one prompt, in portions shorter than the
    convolution, around multiples of eight rows and token by token.  The oracle is checked for showing a lost state, a lost convolution input,
    a state read before the row joins it, and a rule that only adds (rows come back with the same key: their values must be replaced)."""
    for taps, kw in ((4, dict(heads=6, kv_heads=2, dim=12, vdim=9)), (6, dict(heads=2, kv_heads=2, dim=40, vdim=20)), (1, dict(heads=3, kv_heads=1, dim=33, vdim=35))):
        cfg = DC.config(layers=[DC.pair(r=DC.right(conv=taps, a1_rank=4, g1_rank=6, **kw), right_scale=1.2)])
        w = DC.random_tensors(cfg, seed=33 + taps)
        pre = "l0.mix.right."
        m, n, W, eps = cfg["layers"][0]["mixer"]["right"], 300, cfg["width"], cfg["norm"]["eps"]
        H, Dm = m["heads"], m["dim"]
        w[pre + "dt_bias"] = torch.linspace(-9.0, 1.0, H * Dm).view(Dm, H).t().reshape(-1).to(torch.bfloat16).float()        # every head has slow and fast channels
        w[pre + "A_log"] = torch.linspace(-1.0, 0.5, H).to(torch.bfloat16).float()
        if getattr(make, "rounded", False):
            for k in ("k", "k.conv"):
                w[pre + k] = (w[pre + k.replace("k", "q", 1)] + 0.25 * w[pre + k]).to(torch.bfloat16).float()
        h = torch.randn(n, W, generator=torch.Generator().manual_seed(7))
        h[40:] = h[torch.arange(40, n) % 40]               # rows come back: the same keys with the same values
        h[100:140] = h[100:140].flip(0)
        h[2] *= 20.0
        h = h.to(torch.bfloat16).float()
        p64 = _sub64(w, pre)
        run64 = lambda p=p64, rows=h, start=0: D.gated_delta_rule(rows[start:].double(), p, m, eps, D.new_delta_state(m))
        want = 1.2 * run64()
        assert _size(1.2 * run64(start=150)[0] - want[150]) > 0.1 * _size(want[150])
        if taps > 1:
            assert _size(1.2 * run64(dict(p64, **{"k.conv": torch.cat([torch.zeros_like(p64["k.conv"][:, :1]), p64["k.conv"][:, 1:]], 1)}))[5:] - want[5:]) > 0.05 * _size(want[5:])
        real = D.delta_update
        for fault in (lambda S, g, k, v, b: g[:, None] * S + torch.outer(k, b * v), lambda S, g, k, v, b: S + torch.outer(k, b * (v - S.T @ k)),
                      lambda S, g, k, v, b: g[:, None] * S + torch.outer(k, b * (v - S.T @ k))):
            D.delta_update = fault
            try:
                moved = 1.2 * run64()
            finally:
                D.delta_update = real
            assert _size(moved[200:] - want[200:]) > 0.02 * _size(want[200:]), _size(moved[200:] - want[200:]) / _size(want[200:])
        for cut in ((300,), (2, 1, 3, 1, 1, 56, 2, 5, 128, 64) + (1,) * 37, (8, 16, 7, 9, 24, 236)):
            eng = make(cfg, w)
            got = _in_portions(eng, n, cut, [0], lambda model, lo, hi, c: _right_alone(model, h[lo:hi])(c))
            large = [t for t in range(n) if 2 <= t < 2 + taps]                 # the rows whose convolution sees it
            rest = [t for t in range(n) if t not in large]
            _close(got[rest], want[rest], tol, f"gated delta rule, {taps} taps, portions {cut[:3]}...")
            _close(got[large], want[large], tol, f"gated delta rule, {taps} taps, rows of the large input, portions {cut[:3]}...")


def delta_rows_of_several_sequences(make, tol):
    """Rows of four sequences in one launch -- one that starts, two that go on with one and two rows (shorter than the convolution), one with
    many -- against each alone: blocks of eight rows that hold the ends and beginnings of several sequences, for the convolution and the scan."""
    from lmdeploy_b200.turbomind.hybrid import StepArrays
    cfg = DC.config(layers=[DC.pair(DC.left(heads=2, kv_heads=1), r=DC.right(heads=64, kv_heads=32, dim=16, vdim=16, conv=4))])
    w = _weights(make, cfg, seed=51)
    m, eps, pre = cfg["layers"][0]["mixer"]["right"], cfg["norm"]["eps"], "l0.mix.right."
    eng = make(cfg, w)
    dev = eng.model.device
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    first, second = (37, 5, 2, 3), (5, 1, 2, 310)
    g = torch.Generator().manual_seed(5)
    rows = [torch.randn(a + b, cfg["width"], generator=g).to(torch.bfloat16).float() for a, b in zip(first, second)]
    for slot in range(4):
        eng.state.reset(slot)
    got, at = [[] for _ in rows], [0] * 4
    for counts in (first, second):
        h = torch.cat([r[a:a + c] for r, a, c in zip(rows, at, counts)])
        cu = np.concatenate([[0], np.cumsum(counts)])
        c = StepArrays(n=int(cu[-1]), batch=4, tok_seq=i32(np.repeat(range(4), counts)), tok_pos=i32(np.concatenate([np.arange(a, a + k) for a, k in zip(at, counts)])),
                       cu_q=i32(cu), seq_slot=i32([2, 0, 3, 1]), state=eng.state, max_pos=0)
        y = _right_alone(eng.model, h)(c).float().cpu()
        for s in range(4):
            got[s].append(y[cu[s]:cu[s + 1]])
            at[s] += counts[s]
    for s in range(4):
        want = 1.2 * D.gated_delta_rule(rows[s].double(), _sub64(w, pre), m, eps, D.new_delta_state(m))
        _close(torch.cat(got[s]), want, tol, f"sequence {s} of a batch")


def low_rank_rate_decays(make, tol):
    """exp(-rate softplus(z)) for z from far below to far above zero and rates from a thousandth to thirty: decays of nearly one keep their
    distance from one, fast ones vanish without a fault; many rows and few, odd and even channel counts."""
    from lmdeploy_b200 import _hybrid_lib as H
    cfg = DC.config()
    model = make(cfg, DC.random_tensors(cfg)).model
    dev, T = model.device, model.T
    g = torch.Generator().manual_seed(4)
    for n, heads, dim, rank in ((3, 3, 11, 5), (700, 16, 128, 9), (2500, 1, 257, 64)):
        low = torch.randn(n, rank + 3, generator=g).to(torch.bfloat16).float()
        a = torch.randn(heads * dim, rank, generator=g).to(torch.bfloat16).float() / 4
        b = torch.linspace(-20.0, 20.0, heads * dim)
        rate = torch.exp(torch.linspace(-7.0, 3.4, heads))
        z = low[:, :rank].double() @ a.double().T + b.double()
        want = torch.exp(-rate.double().repeat_interleave(dim) * D.softplus(z))
        out = torch.empty(n, heads * dim, dtype=torch.float32, device=dev)
        lo, aw, bw, rw = low.to(dev, T).contiguous(), a.t().to(dev, T).contiguous(), b.to(dev), rate.to(dev)
        H.check(model.lib.b200h_low_rank_rate_decay(lo.data_ptr(), rank + 3, aw.data_ptr(), bw.data_ptr(), rw.data_ptr(), n, heads, dim, rank, out.data_ptr(),
                                                    model.dt, model._stream()))
        _close(out.cpu(), want, 2e-6, f"decays {n} x {heads} x {dim}")
        slow = want > 1 - 1e-3
        if slow.any():
            _close(1.0 - out.cpu().double()[slow], 1.0 - want[slow], 1e-3, "distance from one")


def unit_vectors_and_step_sizes(make, tol):
    """What the gated delta rule reads: queries and keys of zero (stay zero), of the size of the root of 1e-6 (where the added constant counts)
    and large; the scaled dot product of every head; step sizes at large arguments."""
    from lmdeploy_b200 import _hybrid_lib as H
    G, Dm, heads, V = 3, 10, 6, 4
    cfg = DC.config()
    eng = make(cfg, DC.random_tensors(cfg))
    model = eng.model
    dev, T, n, ch = model.device, model.T, 21, 2 * G * Dm + heads * V
    u = torch.randn(n, ch + heads, generator=torch.Generator().manual_seed(3))
    for t, f in ((0, 0.0), (1, 2e-3), (2, 2e-4), (3, 40.0)):
        u[t, :ch] *= f
    u[4, ch:] = 60.0
    u[5, ch:] = -60.0
    u = u.to(torch.bfloat16).float()
    c = _step_arrays(eng, 0, n, [0], slot=0)
    f32 = dict(dtype=torch.float32, device=dev)
    ud, conv, st = u.to(dev, T).contiguous(), torch.ones(1, ch, **f32), torch.zeros(4, 8, **f32)
    qkv, kq, beta = torch.empty(n, ch, **f32), torch.empty(n, G, **f32), torch.empty(n, heads, **f32)
    a = H.DeltaArgs()
    a.n, a.batch, a.heads, a.kv_heads, a.dim, a.vdim, a.taps, a.q_scale, a.unit_eps = n, 1, heads, G, Dm, V, 1, Dm ** -0.5, 1e-6
    a.u, a.b, a.ld, a.conv, a.conv_state, a.slot_stride = ud.data_ptr(), ud.data_ptr() + ud.element_size() * ch, ch + heads, conv.data_ptr(), st.data_ptr(), 8
    a.qkv, a.kq, a.beta = qkv.data_ptr(), kq.data_ptr(), beta.data_ptr()
    a.tok_seq, a.cu_q, a.seq_slot, a.dtype, a.stream = c.tok_seq.data_ptr(), c.cu_q.data_ptr(), c.seq_slot.data_ptr(), model.dt, model._stream()
    H.check(model.lib.b200h_delta_prep(C.byref(a)))
    y = D.silu(u[:, :ch].double())
    q, k = (D.unit_vector(y[:, i * G * Dm:(i + 1) * G * Dm].reshape(n, G, Dm)) for i in range(2))
    q = q * Dm ** -0.5
    assert 0.05 < _size(q[2]) * Dm ** 0.5 < 0.9 and _size(q[0]) == 0                 # the cases are what they are meant to be
    _close(qkv.cpu()[:, :G * Dm], q.reshape(n, -1), 5e-6, "unit queries")
    _close(qkv.cpu()[:, G * Dm:2 * G * Dm], k.reshape(n, -1), 5e-6, "unit keys")
    _close(qkv.cpu()[:, 2 * G * Dm:], y[:, 2 * G * Dm:], 5e-6, "values")
    for t in (1, 2):
        _close(qkv.cpu()[t, :G * Dm], q[t].reshape(-1), 2e-5, "small unit queries")
    _close(kq.cpu(), (q * k).sum(-1), 5e-6, "dot products")
    _close(beta.cpu(), D.sigmoid(u[:, ch:].double()), 5e-6, "step sizes")


def streams_alone(make, tol):
    """The streams' operators for every number of streams, widths for vector and for scalar accesses: the normed embedding copied to all; a
    join that updates all streams from the old ones (a matrix indexed [from, to]: its transpose moves the answer) and feeds the next norm; a
    join over chosen rows that writes nothing; the plain sum; outputs far larger and far smaller than the streams."""
    from lmdeploy_b200 import _hybrid_lib as H
    for W in (48, 33):
        for S in range(1, H.MAX_STREAMS + 1):
            cfg = DC.config(layers=[DC.attention(mlp=DC.dense())], width=W, streams=S)
            w = DC.random_tensors(cfg, seed=37 + S)
            model = make(cfg, w).model
            n, eps, dev, T, mw = 37, cfg["norm"]["eps"], model.device, model.T, model.w
            g = torch.Generator().manual_seed(9)
            rnd = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).float()
            x0, y = rnd(n, S, W), rnd(n, W)
            y[3] *= 64.0
            y[4] /= 64.0
            hc = {k: w["l0.hc1." + k].double() for k in ("in", "out", "mix")}
            xs = [x0[:, s].double() for s in range(S)]
            new = D.write_streams(xs, hc["mix"], hc["out"], y.double() * w["l0.ls1"].double())
            if S > 1:
                other = D.write_streams(xs, hc["mix"].T, hc["out"], y.double() * w["l0.ls1"].double())
                assert _size(torch.stack(other, 1)[5:] - torch.stack(new, 1)[5:]) > 0.01 * _size(torch.stack(new, 1)[5:])
            x, yd = x0.clone().to(dev).contiguous(), y.to(dev, T).contiguous()
            h = torch.empty(n, W, dtype=T, device=dev)
            rows = torch.tensor([4, 0, 36, 4], dtype=torch.int32, device=dev)
            part, total = torch.empty(4, W, dtype=T, device=dev), torch.empty(n, W, dtype=torch.float32, device=dev)
            ptr = lambda t: None if t is None else t.data_ptr()

            def join(y_, read, norm, rows_, count, write, u, out):
                H.check(model.lib.b200h_join_streams(
                    x.data_ptr(), S, ptr(y_), mw["l0.ls1"].data_ptr(), mw["l0.hc1.mix"].data_ptr(), mw["l0.hc1.out"].data_ptr(), ptr(read), ptr(norm),
                    ptr(rows_), count, W, eps, write, ptr(u), ptr(out), model.dt, model._stream()))

            join(yd, None, mw["final.norm"], rows, 4, 0, None, part)
            _close(x.cpu(), x0, 0.0, "a join that writes nothing")
            _close(part.float().cpu(), D.norm(sum(new), w["final.norm"].double(), eps)[[4, 0, 36, 4]], tol, f"{S} streams of {W}: chosen rows")
            join(yd, mw["l0.hc2.in"], mw["l0.norm2"], None, n, 1, None, h)
            for t in range(n):
                _close(x.cpu()[t], torch.stack(new, 1)[t], 2e-6, f"{S} streams of {W}: streams of row {t}")
            want = D.norm(D.read_streams(new, w["l0.hc2.in"].double()), w["l0.norm2"].double(), eps)
            _close(h.float().cpu(), want, tol, f"{S} streams of {W}: next norm")
            join(None, None, None, None, n, 1, total, None)
            _close(total.cpu(), sum(new), 2e-6, f"{S} streams of {W}: sum")
            tokens = torch.tensor([5, 0, 60, 5], dtype=torch.int32, device=dev)
            x = torch.empty(4, S, W, dtype=torch.float32, device=dev)
            H.check(model.lib.b200h_embed_streams(tokens.data_ptr(), mw["embed"].data_ptr(), 1.0, mw["embed.norm"].data_ptr(), x.data_ptr(), S,
                                                  mw["l0.hc1.in"].data_ptr(), mw["l0.norm1"].data_ptr(), 4, W, eps, h.data_ptr(), model.dt, model._stream()))
            e = D.norm(w["embed"].double()[[5, 0, 60, 5]], w["embed.norm"].double(), eps)
            for s in range(S):
                _close(x.cpu()[:, s], e, 2e-6, f"{S} streams of {W}: embedding in stream {s}")
            _close(h[:4].float().cpu(), D.norm(hc["in"].sum() * e, w["l0.norm1"].double(), eps), tol, f"{S} streams of {W}: first norm")


def gated_feed_forward_alone(make, tol):
    """The gelu-gated feed-forward alone, inner sizes that are and are not multiples of four, arguments far below and above zero."""
    for ff in (40, 37):
        cfg = DC.config(layers=[DC.attention(mlp=DC.dense(ff=ff))])
        w = DC.random_tensors(cfg, seed=35)
        h = 2.0 * torch.randn(50, cfg["width"], generator=torch.Generator().manual_seed(9))
        h[1] *= 30.0
        h = h.to(torch.bfloat16).float()
        model = make(cfg, w).model
        got = model.dense_mlp(0, h.to(model.device, model.T).contiguous()).float().cpu()
        want = D.gated_ff(h.double(), _sub64(w, "l0.mlp."))
        rest = [t for t in range(50) if t != 1]
        _close(got[rest], want[rest], tol, f"feed-forward of {ff}")
        _close(got[1], want[1], tol, f"feed-forward of {ff}, large row")


MECHANISMS = [low_rank_rate_decays, unit_vectors_and_step_sizes, streams_alone, gated_feed_forward_alone, delta_rows_of_several_sequences,
              gated_delta_rule_in_portions, retention_in_portions, marked_keys_chunks_and_sinks, marked_keys_windows_and_first_tokens]
ENGINE = [score_scratch_in_row_chunks, whole_prompt, layer_by_layer, prefill_then_decode, token_by_token, portions, unequal_batch,
          left_out_and_resumed, reuse_of_pages_and_slots, other_sizes, wider_sizes, greedy_generation]
ALL = MECHANISMS + ENGINE

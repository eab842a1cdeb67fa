"""Duparax decoders without a GPU: the host side (spec parsing, state and cache offsets, page / slot / row addressing of
turbomind/hybrid.py and the engine) runs the scenarios of tests/duparax_scenarios.py with the numpy stand-in for the CUDA
library, in float32, against the float64 oracle; and the oracle's own mechanisms are checked on cases worked by hand."""
import math

import pytest
import torch

import duparax_cases as DC
import duparax_scenarios as S
from oracle import duparax as D

one = lambda x: torch.tensor(x, dtype=torch.float64)


def _make(cfg, tensors, **kw):
    return DC.build_engine(cfg, tensors, device="cpu", dtype="f32", emulate=True, **kw)


@pytest.mark.parametrize("scenario", S.ALL, ids=lambda f: f.__name__)
def test_engine_scenario_on_the_emulated_library(scenario):
    # whole decoders: unit norms over heads of a few channels amplify the rounding of 32-bit sums; each mechanism alone is tighter
    scenario(_make, 2e-5 if scenario in S.MECHANISMS else 1e-4)


def test_spec_reads_every_size_from_the_config():
    cfg = DC.config()
    spec = DC.spec_of(cfg)
    assert [l.mixer.kind for l in spec.layers] == ["paired", "rglru", "paired", "rglru", "paired"] and spec.block == "sandwich" and spec.plain_norms
    assert (spec.width, spec.vocab, spec.norm_eps, spec.logit_scale) == (48, 61, 1e-5, 0.7)
    assert spec.layers[2].mlp is None and (spec.layers[1].mlp.kind, spec.layers[1].mlp.ff, spec.layers[1].mlp.act) == ("dense", 40, "silu_gate")
    f = spec.layers[0].mlp
    assert (f.experts, f.top, f.ff, f.score, f.act, f.router_bias, f.shared, f.grouped) == (6, 2, 24, "softmax_chosen", "silu_gate", True, 20, False)
    assert spec.layers[3].mlp.shared == 0
    a = spec.layers[2].mixer.left
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.span, a.q_temp, a.rot) == (4, 1, 12, 6, 0.3, 0, None, None)
    assert a.bias and not (a.qk_norm or a.head_norm or a.distance_bias or a.talking_heads or a.gate or a.sink)
    assert spec.layers[4].mixer.left.q_temp == (0.9, 5.0)
    r = spec.layers[4].mixer.right
    assert (r.heads, r.dim, r.vdim, r.rank, r.tau) == (4, 33, 4, 8, 1.5)
    u = spec.layers[3].mixer
    assert (u.width, u.blocks, u.conv_taps, u.rate) == (60, 5, 2, 8.0)
    # the decay's inner size from a tensor's shape when the config does not carry it
    bare = DC.config()
    for e in bare["layers"]:
        if e["type"] == "parallel":
            del e["mixer"]["right"]["rank"]
    from lmdeploy_b200.turbomind.specs import duparax_spec
    assert duparax_spec(bare, tensor_shapes={f"l{i}.mix.right.a1": (9 + i, 48) for i in (0, 2, 4)}).layers[4].mixer.right.rank == 13
    for bad in ([DC.pair(DC.left(heads=5, kv_heads=2))], [DC.rglru(width=10, blocks=3)], [DC.pair(mlp=DC.moe(experts=3, top=4))],
                [DC.pair(DC.left(q_temp=(1.0, 0)))]):
        with pytest.raises(ValueError):
            DC.spec_of(DC.config(layers=bad))
    with pytest.raises(ValueError):
        duparax_spec(bare)
    with pytest.raises(NotImplementedError):
        DC.spec_of(DC.config(layers=[{"type": "attention", "mixer": {}, "mlp": None}]))
    with pytest.raises(NotImplementedError):
        DC.spec_of(DC.config(layers=[DC.pair(mlp={"kind": "tree"})]))


def test_state_and_cache_geometry():
    cfg = DC.config()
    w = DC.random_tensors(cfg)
    model = _make(cfg, w).model
    at, want_conv, want_mix = 0, {}, {}
    for r, e in enumerate(cfg["layers"]):
        m = e["mixer"]
        if e["type"] == "rglru":
            want_conv[r], want_mix[r] = at, at + (m["conv"] - 1) * m["width"]
            at = want_mix[r] + m["width"]
        else:
            at = (at + 3) // 4 * 4
            want_mix[r] = at
            at += m["right"]["heads"] * m["right"]["dim"] * m["right"]["vdim"]
    assert model.mix_off == want_mix and model.slot_floats == at and {k: model.conv_off[k] for k in want_conv} == want_conv
    lefts = [e["mixer"]["left"] for e in cfg["layers"] if e["type"] == "parallel"]
    assert model.block_bytes == sum(64 * m["kv_heads"] * (m["dim"] + m["vdim"]) * 4 for m in lefts)      # float32 keys and values of the attention sides
    assert model.w["l0.in"].shape == (6 * 8 + 3 * 8 + 3 * 10 + 2 * 36 + 2 * 21 + 5, 48) and "l0.left.in" not in model.w
    assert model.w["l3.gates"].shape == (5, 24, 12) and "l2.norm2" not in model.w and model.w["l0.router.b"].shape == (6,)
    assert torch.equal(model.w["l0.norm1b"].cpu(), w["l0.norm1b"])                           # plain weights: nothing is added
    assert torch.allclose(model.w["final.norm"].cpu(), 0.7 * w["final.norm"])                # carries the logit scale


# ------------------------------------------------------------------------------------------------ the oracle on hand-worked cases
def test_oracle_attention_and_growing_queries():
    t = {"coef": 0.5, "every": 4}
    assert [D.query_growth(p, t) for p in (0, 2, 3, 6, 7)] == [1.0, 1.0, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3)]
    assert D.query_growth(99, None) == 1.0
    # one head of one dimension, q = k = 1 from biases, values = the input: the mean of all earlier values, projected by 2
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0}
    p = {"q": one([[0.0]]), "k": one([[0.0]]), "v": one([[1.0]]), "q.b": one([1.0]), "k.b": one([1.0]), "v.b": one([0.5]), "o": one([[2.0]])}
    out = D.attention(one([[1.0], [3.0], [8.0]]), p, m, [0, 1, 2], D.new_attention_state(m))
    assert torch.allclose(out.reshape(-1), one([3.0, 5.0, 9.0]))
    # keys = the input: a query at a position where it has grown divides the weights as its larger scores say
    p = dict(p, k=one([[1.0]]), **{"k.b": one([0.0]), "v.b": one([0.0])})
    out = D.attention(one([[math.log(2.0)], [0.0]]), p, dict(m, q_temp={"coef": 1.0 / math.log(2.0), "every": 2}), [0, 1], D.new_attention_state(m))
    assert abs(float(out[1, 0]) - 2.0 * math.log(2.0) * 4.0 / 5.0) < 1e-12                    # score 2 ln 2: weights 4/5 and 1/5


def test_oracle_gated_linear_attention_of_one_head():
    m = {"heads": 1, "dim": 1, "vdim": 1, "tau": 2.0}
    p = {"q": one([[1.0]]), "k": one([[1.0]]), "v": one([[1.0]]), "g": one([[50.0]]), "a1": one([[0.0]]), "a2": one([[0.0]]),
         "a2.b": one([-math.log(3.0)]), "norm": one([3.0]), "o": one([[1.0]])}
    assert abs(float(D.channel_decays(one([5.0]), p, m)[0, 0]) - 0.5) < 1e-12                # sigmoid = 1/4, its square root
    st = D.new_linear_state(m)
    out = D.gated_linear_attention(one([[1.0], [2.0]]), p, m, 0.0, st)
    assert abs(float(st["S"][0, 0, 0]) - (0.5 * 1.0 + 4.0)) < 1e-12                           # the row itself has joined the state
    assert torch.allclose(out.reshape(-1), one([150.0, 300.0]))                              # unit norm, weight 3, silu(50 h) ~ 50 h
    m2 = {"heads": 1, "dim": 4, "vdim": 1, "tau": 1.0}
    p2 = {"q": torch.ones(4, 1, dtype=torch.float64), "k": torch.ones(4, 1, dtype=torch.float64), "v": one([[1.0]]), "g": one([[0.0]]),
          "a1": one([[0.0]]), "a2": torch.zeros(4, 1, dtype=torch.float64), "a2.b": torch.zeros(4, dtype=torch.float64), "norm": one([1.0]), "o": one([[1.0]])}
    st = D.new_linear_state(m2)
    D.gated_linear_attention(one([[2.0]]), p2, m2, 0.0, st)
    assert st["S"].reshape(-1).tolist() == [4.0] * 4


def test_oracle_real_gated_recurrence():
    m = {"width": 2, "blocks": 2, "conv": 2}
    z2 = torch.zeros(2, dtype=torch.float64)
    p = {"y": torch.zeros(2, 1, dtype=torch.float64), "y.b": one([30.0, 30.0]), "x": one([[1.0], [2.0]]), "x.b": one([0.5, 0.0]),
         "conv": one([[0.0, 1.0], [1.0, 0.0]]), "conv.b": one([0.0, 0.25]), "ra": torch.zeros(2, 1, 1, dtype=torch.float64), "ra.b": torch.zeros(2, 1, dtype=torch.float64),
         "ri": torch.zeros(2, 1, 1, dtype=torch.float64), "ri.b": torch.full((2, 1), 40.0, dtype=torch.float64), "lam": z2, "o": torch.eye(2, dtype=torch.float64)}
    out = D.rglru(one([[1.0], [3.0]]), p, m, D.new_rglru_state(m))
    a = math.exp(-8.0 * 0.5 * math.log(2.0))                                                  # 1/16
    s = math.sqrt(1 - a * a)
    # u: channel 0 takes the current input + 0.5; channel 1 the previous one (zero before the start) + 0.25
    want = [[s * 1.5 * 30, s * 0.25 * 30], [(a * s * 1.5 + s * 3.5) * 30, (a * s * 0.25 + s * 2.25) * 30]]
    assert torch.allclose(out, one(want))
    r, i = D.rglru_gates(one([1.0, 2.0, 3.0, 4.0]), {"ra": one([[[0.0, 1.0], [0.0, 0.0]], [[0.0, 0.0], [1.0, 0.0]]]), "ra.b": torch.zeros(2, 2, dtype=torch.float64),
                                                     "ri": torch.zeros(2, 2, 2, dtype=torch.float64), "ri.b": torch.zeros(2, 2, dtype=torch.float64)}, 2)
    assert torch.allclose(r, D.sigmoid(one([2.0, 0.0, 0.0, 3.0]))) and i.tolist() == [0.5] * 4


def test_oracle_router_and_activation():
    f = {"router": {"experts": 3, "top": 2}}
    p = {"router": one([[0.0], [1.0], [2.0]]), "router.b": one([1.5, 0.0, 0.0])}
    (e0, w0), (e1, w1) = D.route(one([1.0]), p, f)
    assert (e0, e1) == (2, 0) and abs(float(w0) - 1 / (1 + math.exp(-0.5))) < 1e-12 and abs(float(w0 + w1) - 1) < 1e-12
    assert torch.allclose(D.gelu_tanh(one([1.0, -1.0])), one([0.841191990608, -0.158808009392]))
    assert torch.allclose(D.gated_ff(one([[2.0]]), {"gate": one([[1.0]]), "up": one([[3.0]]), "down": one([[1.0]])}), one([[2 / (1 + math.exp(-2.0)) * 6]]))


def test_bench_configuration_builds_a_spec():
    """The sizes bench.py --hybrid-design duparax runs parse into a spec whose tensors have the expected shapes."""
    import bench
    from lmdeploy_b200.turbomind.hybrid import HybridModel
    from lmdeploy_b200.turbomind.specs import duparax_spec
    for size, z in bench.HYBRID_SIZES.items():
        spec = duparax_spec(bench.duparax_bench_config(z), name=size)
        assert [l.mixer.kind for l in spec.layers] == ["paired", "paired", "rglru", "paired"] and spec.layers[0].mlp.kind == "dense"
        shapes = HybridModel.tensor_shapes(DC._Shapes(spec))
        W = z["width"]
        assert shapes["l0.mix.right.a1"] == (64, W) and shapes["l2.mix.ra"] == (16, W // 16, W // 16) and shapes["l3.mlp.shared.down"] == (W, z["ff"])

"""Sefuvik decoders without a GPU: the host side (spec parsing, state and cache offsets, page / slot / row addressing of
turbomind/hybrid.py and the engine) runs the scenarios of tests/sefuvik_scenarios.py with the numpy stand-in for the CUDA
library, in float32, against the float64 oracle; and the oracle's own mechanisms are checked on cases worked by hand."""
import copy
import math

import pytest
import torch

import sefuvik_cases as DC
import sefuvik_scenarios as S
from oracle import sefuvik as D

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
    assert [l.mixer.kind for l in spec.layers] == ["window_attention", "retention", "paired", "paired", "retention", "window_attention"]
    assert (spec.block, spec.width, spec.vocab, spec.norm_eps, spec.streams, spec.tied_head, spec.plain_norms) == ("streams", 48, 61, 1e-5, 3, True, False)
    assert spec.layers[1].mlp is None and (spec.layers[0].mlp.ff, spec.layers[0].mlp.act) == (40, "gelu_gate")
    a = spec.layers[5].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.keep_first, a.maps, a.diff, a.chunk) == (4, 1, 12, 8, 0.3, 90, 7, 2, 0.6, 0)
    assert a.bias and not (a.qk_norm or a.head_norm or a.distance_bias or a.talking_heads or a.gate or a.sink) and a.rot is None
    assert (a.span, a.q_cols, a.k_cols, a.v_cols, a.proj_cols) == (97, 96, 24, 8, 128)
    r = spec.layers[4].mixer
    assert (r.heads, r.dim, r.vdim, r.decay, r.rot.dims, r.rot.base, r.rot.halves) == (2, 33, 20, (0.5, 0.998), 32, 500.0, True)
    l, g = spec.layers[3].mixer.left, spec.layers[3].mixer.right
    assert (l.heads, l.kv_heads, l.dim, l.vdim, l.chunk, l.window, l.sink, l.gate, l.gate_per_head, l.bias) == (3, 1, 6, 14, 70, 0, True, True, False, False)
    assert (g.heads, g.kv_heads, g.dim, g.vdim, g.conv_taps, g.decay_rank, g.gate_rank) == (3, 3, 7, 33, 2, 8, 6) and spec.layers[3].mixer.scales == (1.3, 0.6)
    # the low-rank matrices' inner sizes from tensor shapes when the config does not carry them
    bare = copy.deepcopy(cfg)
    for e in bare["layers"]:
        if e["type"] == "parallel":
            del e["mixer"]["right"]["a1_rank"], e["mixer"]["right"]["g1_rank"]
    from lmdeploy_b200.turbomind.specs import sefuvik_spec
    g = sefuvik_spec(bare, tensor_shapes={f"l{i}.mix.right.{k}": (9 + i + j, 48) for i in (2, 3) for j, k in enumerate(("a1", "g1"))}).layers[3].mixer.right
    assert (g.decay_rank, g.gate_rank) == (12, 13)
    with pytest.raises(ValueError):
        sefuvik_spec(bare)
    for bad in ([DC.attention(heads=5, kv_heads=2)], [DC.pair(DC.left(heads=5, kv_heads=2))], [DC.pair(r=DC.right(heads=3, kv_heads=2))],
                [DC.retention(decay=(0.5,))], [DC.retention(dims=7)], [DC.retention(dims=14)], [DC.pair(DC.left(dims=12))]):
        with pytest.raises(ValueError):
            DC.spec_of(DC.config(layers=bad))
    for bad in ([{"type": "rglru", "mixer": {}, "mlp": None}], [DC.attention(mlp={"kind": "moe"})]):
        with pytest.raises(NotImplementedError):
            DC.spec_of(DC.config(layers=bad))


def test_state_and_cache_geometry():
    cfg = DC.config()
    w = DC.random_tensors(cfg)
    model = _make(cfg, w).model
    up4 = lambda v: (v + 3) // 4 * 4
    at, page, conv, mix = 0, 0, {}, {}
    for r, e in enumerate(cfg["layers"]):
        m = e["mixer"]
        if e["type"] == "retention":
            mix[r] = at = up4(at)
            at += m["heads"] * m["dim"] * m["vdim"]
        elif e["type"] == "parallel":
            g = m["right"]
            conv[r] = at
            at += (g["conv"] - 1) * (2 * g["kv_heads"] * g["dim"] + g["heads"] * g["vdim"])
            mix[r] = at = up4(at)
            at += g["heads"] * g["dim"] * g["vdim"]
            page += 64 * m["left"]["kv_heads"] * (m["left"]["dim"] + m["left"]["vdim"]) * 4
        else:
            page += 64 * m["kv_heads"] * (2 * m["dim"] + m["vdim"]) * 4                       # two keys per value
    assert model.mix_off == mix and {k: model.conv_off[k] for k in conv} == conv and model.slot_floats == up4(at) and model.block_bytes == page
    # one product feeds both sides of a pair, every part from a multiple of eight columns on; one output product takes both
    l, g = cfg["layers"][2]["mixer"]["left"], cfg["layers"][2]["mixer"]["right"]
    cols = model.w["l2.cols"]
    assert all(v % 8 == 0 for v in cols.values()) and cols["u"] >= (4 + 2) * 10 + 2 * 6 + 4 * 6 and model.w["l2.in"].shape[1] == 48
    assert model.w["l2.o"].shape == (48, (4 * 6 + 4 * 9 + 7) // 8 * 8) and torch.equal(model.w["l2.o"][:, :24].cpu(), w["l2.mix.left.o"])
    assert torch.equal(model.w["l2.in"][cols["g1"]:cols["g1"] + 3].cpu(), w["l2.mix.right.g1"])
    assert torch.allclose(model.w["l2.right.norm"].cpu(), 1.2 * w["l2.mix.right.norm"].repeat(4))           # carries the side's scale
    assert torch.equal(model.w["l2.right.conv"].cpu().t(), torch.cat([w[f"l2.mix.right.{k}.conv"] for k in "qkv"]))
    for name in ("embed.norm", "l0.norm1", "final.norm"):
        assert torch.allclose(model.w[name].cpu(), 1.0 + w[name])
    want = D.subtraction_factor({k: w["l0.mix." + k].double() for k in ("lq1", "lk1", "lq2", "lk2")}, cfg["layers"][0]["mixer"])
    assert abs(model.w["l0.lambda"] - float(want)) < 1e-12
    assert "l1.norm2" not in model.w and "l1.hc2.mix" not in model.w
    with pytest.raises(ValueError):
        _make(cfg, dict(w, **{"l0.mix.lq1": w["l0.mix.lq1"][:3]}))
    for kw in (dict(streams=9), dict(layers=[DC.retention(heads=1, dim=300, decay=(0.5,))]), dict(layers=[DC.pair(r=DC.right(conv=17))])):
        with pytest.raises(NotImplementedError):
            bad = DC.config(**kw)
            _make(bad, DC.random_tensors(bad))


# ------------------------------------------------------------------------------------------------ the oracle on hand-worked cases
def test_oracle_windows_and_chunks():
    assert D.window_keys(10, 4, 2) == [0, 1, 7, 8, 9, 10] and D.window_keys(3, 4, 2) == [0, 1, 2, 3] and D.window_keys(4, 4, 0) == [1, 2, 3, 4]
    assert D.window_keys(5, 1, 9) == [0, 1, 2, 3, 4, 5]
    assert D.chunk_keys(7, 4) == [4, 5, 6, 7] and D.chunk_keys(8, 4) == [8] and D.chunk_keys(2, 4) == [0, 1, 2]


def test_oracle_rotation_of_halves():
    x = one([[1.0, 2.0, 3.0, 4.0, 5.0]])
    y = D.rotate_halves(x, 3, {"dims": 4, "base": 100.0})
    c0, s0, c1, s1 = math.cos(3.0), math.sin(3.0), math.cos(0.3), math.sin(0.3)
    assert torch.allclose(y, one([[c0 - 3 * s0, 2 * c1 - 4 * s1, 3 * c0 + s0, 4 * c1 + 2 * s1, 5.0]]))
    assert torch.equal(D.rotate_halves(x, 0, {"dims": 4, "base": 100.0}), x)


def test_oracle_differential_attention_of_one_head():
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 2, "scale": 1.0, "mask": None, "diff": 0.2}
    z = one([0.0])
    p = {"q": one([[0.0], [0.0]]), "k": one([[0.0], [1.0]]), "v": one([[1.0], [2.0]]), "q.b": one([0.0, 1.0]), "k.b": one([0.0, 0.0]), "v.b": one([0.0, 0.0]),
         "lq1": one([1.0]), "lk1": one([math.log(1.5)]), "lq2": z, "lk2": z, "o": torch.eye(2, dtype=torch.float64)}
    lam = 1.5 - 1.0 + 0.2
    assert abs(float(D.subtraction_factor(p, m)) - lam) < 1e-12
    # map 1 averages; map 2 has scores ln 3 and 0: weights 3/4 and 1/4
    h = one([[math.log(3.0)], [0.0]])
    out = D.differential_attention(h, p, m, 0.0, [0, 1], D.new_differential_state(m))
    v = math.log(3.0)
    a = (0.5 - lam * 0.75) * v
    assert torch.allclose(out[1], 0.8 * one([a, 2 * a]) / math.sqrt((a * a + 4 * a * a) / 2))


def test_oracle_retention_of_one_head():
    m = {"heads": 1, "dim": 1, "vdim": 1, "decay": [0.5], "rot": {"dims": 0, "base": 1.0}}
    p = {"q": one([[1.0]]), "k": one([[1.0]]), "v": one([[1.0]]), "g": one([[50.0]]), "o": one([[1.0]])}
    st = D.new_retention_state(m)
    out = D.retention(one([[1.0], [2.0]]), p, m, 0.0, [0, 1], st)
    assert abs(float(st["S"]) - 4.5) < 1e-12 and torch.allclose(out.reshape(-1), one([50.0, 100.0]))          # unit norm, silu(50 h) ~ 50 h
    m = dict(m, dim=4)
    p = dict(p, q=torch.ones(4, 1, dtype=torch.float64), k=torch.ones(4, 1, dtype=torch.float64))
    st = D.new_retention_state(m)
    D.retention(one([[2.0]]), p, m, 0.0, [0], st)
    assert st["S"].reshape(-1).tolist() == [2.0] * 4                                                          # k / sqrt(4)


def test_oracle_delta_update_replaces_a_value():
    S0 = torch.zeros(2, 1, dtype=torch.float64)
    k = one([0.6, 0.8])
    S1 = D.delta_update(S0, one([1.0, 1.0]), k, one([5.0]), one(1.0))
    assert abs(float((S1.T @ k)[0]) - 5.0) < 1e-12
    S2 = D.delta_update(S1, one([1.0, 1.0]), k, one([-3.0]), one(1.0))
    assert abs(float((S2.T @ k)[0]) + 3.0) < 1e-12                                                            # not 2: the old value is gone
    S3 = D.delta_update(S1, one([0.5, 1.0]), k, one([1.0]), one(0.5))
    seen = 0.5 * 3.0 * 0.6 + 4.0 * 0.8
    assert torch.allclose(S3.reshape(-1), one([1.5, 4.0]) + k * 0.5 * (1.0 - seen))


def test_oracle_delta_inputs():
    assert torch.allclose(D.unit_vector(one([3e-3, 4e-3])), one([3e-3, 4e-3]) / math.sqrt(25e-6 + 1e-6))
    y, past = D.short_convolution(one([2.0]), one([[10.0, 1.0, 0.5]]), one([[0.0], [3.0]]))
    assert abs(float(y) - 4.0 / (1 + math.exp(-4.0))) < 1e-12 and past.reshape(-1).tolist() == [3.0, 2.0]
    m = {"heads": 2, "dim": 1}
    p = {"a1": one([[1.0]]), "a2": one([[0.0], [0.0]]), "dt_bias": one([0.0, math.log(math.e ** 2 - 1)]), "A_log": one([0.0, math.log(0.5)])}
    assert torch.allclose(D.channel_decays(one([7.0]), p, m).reshape(-1), one([0.5, math.exp(-1.0)]))         # softplus = ln 2, 2


def test_oracle_streams_and_feed_forward():
    xs = [one([[1.0]]), one([[10.0]])]
    new = D.write_streams(xs, one([[1.0, 2.0], [3.0, 4.0]]), one([100.0, 200.0]), one([[1.0]]))
    assert [float(t) for t in new] == [1 + 30 + 100, 2 + 40 + 200]
    assert float(D.read_streams(xs, one([0.5, 0.25]))) == 3.0
    assert torch.allclose(D.gelu_tanh(one([1.0, -1.0])), one([0.841191990608, -0.158808009392]))
    assert torch.allclose(D.norm(one([[3.0, 4.0]]), one([0.0, 1.0]), 0.0), one([[3.0, 8.0]]) / math.sqrt(12.5))


def test_hybrid_structures_match_the_header(tmp_path):
    """The ctypes mirrors that Sefuvik's operators take, against the C header: sizes and every field's offset."""
    import ctypes as C
    import os
    import subprocess
    from lmdeploy_b200 import _hybrid_lib as H
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    pairs = [("b200h_rotary", H.Rotary), ("b200h_window_args", H.WindowArgs), ("b200h_delta_args", H.DeltaArgs), ("b200h_latent_args", H.LatentArgs),
             ("b200h_conv_prep_args", H.ConvPrepArgs)]
    lines = ['#include <stddef.h>', '#include <stdio.h>', '#include "b200_hybrid.h"', 'int main(void) {']
    for cname, cls in pairs:
        lines.append(f'  printf("{cname} %zu\\n", sizeof({cname}));')
        lines += [f'  printf("{cname}.{f[0]} %zu\\n", offsetof({cname}, {f[0].rstrip("_")}));' for f in cls._fields_]
    src, exe = tmp_path / "layout.c", tmp_path / "layout"
    src.write_text("\n".join(lines + ['  return 0;', '}']))
    r = subprocess.run(["gcc", "-std=c99", "-I", os.path.join(root, "include"), str(src), "-o", str(exe)], capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    got = dict(ln.split() for ln in subprocess.check_output([str(exe)], text=True).splitlines())
    for cname, cls in pairs:
        assert int(got[cname]) == C.sizeof(cls), cname
        for f in cls._fields_:
            assert int(got[f"{cname}.{f[0]}"]) == getattr(cls, f[0]).offset, (cname, f[0])


def test_bench_configuration_builds_a_spec():
    """The sizes bench.py --hybrid-design sefuvik runs parse into a spec whose tensors have the expected shapes."""
    import bench
    from lmdeploy_b200.turbomind.hybrid import HybridModel
    from lmdeploy_b200.turbomind.specs import sefuvik_spec
    for size, z in bench.HYBRID_SIZES.items():
        spec = sefuvik_spec(bench.sefuvik_bench_config(z), name=size)
        assert [l.mixer.kind for l in spec.layers] == ["window_attention", "paired", "retention", "paired"] and spec.streams == 4
        shapes = HybridModel.tensor_shapes(DC._Shapes(spec))
        W = z["width"]
        assert shapes["l0.mix.q"] == (z["dense"]["heads"] * 128, W) and shapes["l1.mix.right.a1"] == (64, W) and shapes["l2.mix.g"] == (W, W)

"""Scaffolding of the Sefuvik tests: small configurations with random weights, the engine built on them (on a GPU with the
CUDA library, or on the CPU with tests/hybrid_emulator.py standing in for it) and the same tokens through the plain oracle
(oracle/sefuvik.py, float64).  Schedules are replayed with hybrid_cases.replay."""
import dataclasses

import torch

from hybrid_cases import BLOCK, _Shapes, prompts_for, rel_error, replay  # noqa: F401  (re-exported for the scenarios)
from oracle import sefuvik as D


def attention(heads=6, kv_heads=3, dim=8, vdim=10, scale=0.5, size=37, keep_first=3, diff=0.3, mlp=None):
    mask = {"size": size, "keep_first": keep_first} if size else None
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": mask, "diff": diff}, "mlp": mlp}


def retention(heads=3, dim=12, vdim=7, decay=(0.9, 0.99, 1.0), dims=8, base=500.0, mlp=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"dims": dims, "base": base}}, "mlp": mlp}


def left(heads=4, kv_heads=2, dim=10, vdim=6, scale=0.4, size=41, dims=6, base=2000.0):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size} if size else None,
            "rot": {"dims": dims, "base": base}}


def right(heads=4, kv_heads=2, dim=12, vdim=9, conv=4, a1_rank=5, g1_rank=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "a1_rank": a1_rank, "g1_rank": g1_rank}


def pair(l=None, r=None, left_scale=0.7, right_scale=1.2, mlp=None):
    return {"type": "parallel", "mixer": {"left": l or left(), "right": r or right(), "left_scale": left_scale, "right_scale": right_scale}, "mlp": mlp}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def config(layers=None, width=48, vocab=61, eps=1e-5, streams=3):
    """A Sefuvik config.json as a dict.  The default stack: every mixer, twice, with sizes that are neither equal to each other nor powers of
    two; a layer without a feed-forward; windows and chunks that are not multiples of a page."""
    if layers is None:
        layers = [attention(mlp=dense()), retention(), pair(mlp=dense(ff=28)),
                  pair(left(heads=3, kv_heads=1, dim=6, vdim=14, size=70, dims=6), right(heads=3, kv_heads=3, dim=7, vdim=33, conv=2, a1_rank=8, g1_rank=6),
                       left_scale=1.3, right_scale=0.6),
                  retention(heads=2, dim=33, vdim=20, decay=(0.5, 0.998), dims=32, mlp=dense(ff=24)),
                  attention(heads=4, kv_heads=1, dim=12, vdim=8, scale=0.3, size=90, keep_first=7, diff=0.6, mlp=dense(ff=36))]
    return {"architecture": "Sefuvik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "streams": streams}


def spec_of(cfg):
    from lmdeploy_b200.turbomind.specs import sefuvik_spec
    return sefuvik_spec(cfg)


def random_tensors(cfg, seed=0):
    """name -> float32 tensor with bf16-representable values (so bf16 and float32 engines and the float64 oracle share them)."""
    from lmdeploy_b200.turbomind.hybrid import HybridModel
    shapes = HybridModel.tensor_shapes(_Shapes(spec_of(cfg)))
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        if name.endswith(("norm1", "norm2", "final.norm", "embed.norm")):
            t = 0.3 * torch.randn(shape, generator=g)                           # deviations from one
        elif name.endswith("right.norm"):
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)
        elif name.endswith((".ls1", ".ls2")):
            t = 0.8 + 0.3 * torch.randn(shape, generator=g)
        elif ".hc" in name:
            t = (torch.eye(shape[0]) if len(shape) == 2 else torch.full(shape, 1.0 if name.endswith("out") else 1.0 / shape[0])) \
                + 0.4 * torch.randn(shape, generator=g) / shape[0]
        elif name.endswith("sink"):
            t = torch.randn(shape, generator=g)
        elif name.endswith("A_log"):
            t = torch.log(0.05 + 2.0 * torch.rand(shape, generator=g))
        elif name.endswith("dt_bias"):
            t = -2.0 + 1.5 * torch.randn(shape, generator=g)                    # decays from nearly one to a small fraction
        elif name.endswith("conv"):
            t = torch.randn(shape, generator=g) * (1.0 / shape[-1] ** 0.5)
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = 0.3 * torch.randn(shape, generator=g)
        elif name.endswith(".b") and len(shape) == 1:
            t = 0.3 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * (1.2 / shape[-1] ** 0.5)
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out


def build_engine(cfg, tensors, *, device, dtype="f32", blocks=8, max_batch=4, emulate=False, prefill_tokens=None):
    """TurboMind over a HybridModel holding `tensors`.  emulate: the numpy stand-in replaces the CUDA library (CPU only)."""
    from lmdeploy_b200 import _hybrid_lib as H
    from lmdeploy_b200.messages import TurbomindEngineConfig
    from lmdeploy_b200.turbomind.engine import TurboMind
    from lmdeploy_b200.turbomind.hybrid import HybridModel
    spec = dataclasses.replace(spec_of(cfg), dtype=dtype)
    real = H.load
    if emulate:
        from hybrid_emulator import EmulatedHybridLib
        H.load = lambda: EmulatedHybridLib()
    try:
        model = HybridModel(spec, block_len=BLOCK, max_batch=max_batch, device=device)
    finally:
        H.load = real
    model.load_weights(lambda k: tensors[k])
    ecfg = TurbomindEngineConfig(cache_max_entry_count=blocks, max_batch_size=max_batch,
                                 session_len=blocks * BLOCK + 1, max_prefill_token_num=prefill_tokens or blocks * BLOCK)
    return TurboMind(spec, ecfg, model=model)


def oracle_logits(cfg, tensors, tokens, trace=None):
    """The whole prompt through the plain implementation in float64 -> [n, vocab]."""
    return D.Decoder(cfg, tensors, torch.float64).forward(list(tokens), trace).numpy()

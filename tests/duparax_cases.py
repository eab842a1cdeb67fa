"""Scaffolding of the Duparax tests: small configurations with random weights, the engine built on them (on a GPU with the
CUDA library, or on the CPU with tests/hybrid_emulator.py standing in for it) and the same tokens through the plain oracle
(oracle/duparax.py, float64).  Schedules are replayed with hybrid_cases.replay."""
import dataclasses

import torch

from hybrid_cases import BLOCK, _Shapes, prompts_for, rel_error, replay  # noqa: F401  (re-exported for the scenarios)
from oracle import duparax as D


def left(heads=6, kv_heads=3, dim=8, vdim=10, scale=0.6, q_temp=(0.4, 37)):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if q_temp is not None:
        m["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    return m


def right(heads=3, dim=12, vdim=7, rank=5, tau=4.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "rank": rank, "tau": tau}


def pair(l=None, r=None, mlp=None):
    return {"type": "parallel", "mixer": {"left": l or left(), "right": r or right()}, "mlp": mlp}


def rglru(width=36, blocks=3, conv=4, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def moe(experts=6, top=2, ff=24, shared=20):
    f = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def config(layers=None, width=48, vocab=61, eps=1e-5, logit_scale=0.7):
    """A Duparax config.json as a dict.  The default stack: routed, recurrent, a pair without a feed-forward, recurrent with routed
    experts, a dense pair; sizes that are neither equal to each other nor powers of two, a recurrent branch narrower and one wider than
    the model."""
    if layers is None:
        layers = [pair(mlp=moe()), rglru(mlp=dense()),
                  pair(left(heads=4, kv_heads=1, dim=12, vdim=6, scale=0.3, q_temp=None), right(heads=2, dim=7, vdim=33, rank=3, tau=16.0)),
                  rglru(width=60, blocks=5, conv=2, mlp=moe(experts=4, top=3, ff=16, shared=0)),
                  pair(left(heads=2, kv_heads=2, dim=6, vdim=14, q_temp=(0.9, 5)), right(heads=4, dim=33, vdim=4, rank=8, tau=1.5), mlp=dense(ff=28))]
    return {"architecture": "Duparax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_scale": logit_scale}


def spec_of(cfg):
    from lmdeploy_b200.turbomind.specs import duparax_spec
    return duparax_spec(cfg)


def random_tensors(cfg, seed=0):
    """name -> float32 tensor with bf16-representable values (so bf16 and float32 engines and the float64 oracle share them)."""
    from lmdeploy_b200.turbomind.hybrid import HybridModel
    shapes = HybridModel.tensor_shapes(_Shapes(spec_of(cfg)))
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes.items():
        if name.endswith(("norm1", "norm2", "norm1b", "norm2b", "final.norm", ".norm", ".out")):
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)
        elif name.endswith("a2.b"):
            t = -1.0 + 2.0 * torch.randn(shape, generator=g)                # decays from nearly one to a small fraction
        elif name.endswith(".lam"):
            t = -7.0 + 7.0 * torch.rand(shape, generator=g)                 # a between exp(-8 * 0.7) and 0.993 at r = 1
        elif name.endswith("conv"):
            t = torch.randn(shape, generator=g) * (1.0 / shape[-1] ** 0.5)
        elif name.endswith(".b"):
            t = 0.3 * torch.randn(shape, generator=g)
        elif name.endswith("router"):
            t = torch.randn(shape, generator=g) * (3.0 / shape[-1] ** 0.5)
        elif name == "embed":
            t = 0.5 * torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * (1.5 / shape[-1] ** 0.5)
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

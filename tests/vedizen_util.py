"""Small Vedizen configurations for the tests."""
import copy

import torch

from oracle import vedizen_plain as P
from tests.hybrid_util import TOL, err, save_folder, tokens  # noqa: F401  (shared helpers)


def attn(heads=4, kv_heads=2, dim=24, vdim=40, chunk=37, scale=0.31, softcap=9.0, diff=0.3, mlp=72, limit=1.5):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "scale": scale,
                                           "softcap": softcap, "diff": diff}, "mlp": None if mlp is None else {"kind": "dense", "ff": mlp, "limit": limit}}


def gla(heads=2, dim=20, vdim=28, tau=8.0, mlp=50, limit=0.9):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau},
            "mlp": None if mlp is None else {"kind": "dense", "ff": mlp, "limit": limit}}


def config(layers, width=96, vocab=130, eps=1e-5, scale=3.0, loop=None):
    return {"architecture": "Vedizen", "embedding": {"scale": scale}, "layers": layers, "loop": loop and dict(zip(("start", "stop", "times"), loop)),
            "norm": {"eps": eps}, "vocab": vocab, "width": width}


# layer orders, loops at every place, missing and present feed-forwards, sizes off every alignment, equal and unit values
CONFIGS = {
    "mixed": config([gla(), attn(), gla(3, 48, 72, mlp=None), attn(6, 2, 32, 64, 64, softcap=30.0, mlp=64), gla(2, 64, 128)], loop=(1, 4, 3)),
    "odd": config([attn(3, 1, 9, 11, 5, mlp=13), gla(3, 7, 5, 1.0, mlp=9), attn(2, 2, 7, 13, 33, softcap=80.0, mlp=None)], width=45, vocab=61, eps=1e-3,
                  scale=1.0, loop=(0, 1, 2)),
    "one": config([attn(1, 1, 16, 16, 1, mlp=32), gla(1, 16, 16, mlp=16)], width=32, vocab=40, loop=(0, 2, 1)),
    "wide": config([gla(2, 128, 256, 4.0, mlp=256), attn(12, 1, 128, 128, 70, 0.09, 20.0, mlp=128), gla(4, 32, 64)], width=264, loop=(2, 3, 4)),
    "plain": config([attn(8, 4, 64, 96, 100, 0.125), gla(1, 33, 30)], width=80),
}


def model(name_or_cfg, seed=0, gain=2.0):
    cfg = copy.deepcopy(CONFIGS[name_or_cfg] if isinstance(name_or_cfg, str) else name_or_cfg)
    return cfg, P.random_model(cfg, seed, gain)


def runner_of(cfg, w, dtype):
    from tpp_pytorch_extension_b200.llm import fused_vedizen_infer as FV
    return FV._from_tensors(FV.VedizenShape.from_config(cfg), {k: v.to(torch.bfloat16) for k, v in w.items()}, dtype, "cuda")

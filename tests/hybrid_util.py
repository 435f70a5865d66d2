"""Small configurations of the hybrid decoder for the tests, and helpers around the plain implementation."""
import copy
import json
import os

import torch

from oracle import hybrid_plain as P


def attn(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=28, q_rank=36, window=37, scale=0.31, base=5000.0, kv_from=None, mlp=72):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "mask": {"size": window},
         "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if mlp is None else {"kind": "dense", "ff": mlp}}


def delta(heads=2, dim=20, mlp=None, decay_rank=8):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim, "decay_rank": decay_rank},
            "mlp": None if mlp is None else {"kind": "dense", "ff": mlp}}


def config(layers, width=96, vocab=130, taps=4, eps=1e-5, alpha=1.7):
    return {"architecture": "Dofivik", "canon": {"taps": taps}, "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha, "vocab": vocab,
            "width": width}


# layer orders, sharing, missing and present feed-forwards, sizes off every alignment, equal and unit values
CONFIGS = {
    "mixed": config([attn(), delta(), attn(kv_from=0, window=70, heads=5, vdim=16, scale=0.2), delta(3, 64, mlp=50), attn(window=33, kv_rank=16)]),
    "odd": config([delta(3, 7, decay_rank=5), attn(1, 9, 2, 5, 11, 13, window=5, mlp=13), delta(1, 33, mlp=9), attn(2, 9, 2, 7, 11, 6, window=8, kv_from=1, mlp=None)],
                  width=45, vocab=61, taps=2, eps=1e-3, alpha=1.0),
    "one": config([attn(1, 16, 4, 16, 16, 16, window=1, mlp=32), delta(1, 16)], width=32, vocab=40, taps=1),
    "wide": config([delta(2, 128), attn(4, 128, 64, 128, 512, 192, window=100, scale=0.07, mlp=256), delta(4, 32, mlp=64)], width=256, taps=6),
}


def model(name_or_cfg, seed=0, gain=1.5):
    cfg = copy.deepcopy(CONFIGS[name_or_cfg] if isinstance(name_or_cfg, str) else name_or_cfg)
    return cfg, P.random_model(cfg, seed, gain)


def runner_of(cfg, w, dtype):
    from tpp_pytorch_extension_b200.llm import fused_dofivik_infer as FD
    return FD._from_tensors(FD.DofivikShape.from_config(cfg), {k: v.to(torch.bfloat16) for k, v in w.items()}, dtype, "cuda")


def save_folder(path, cfg, w):
    from tpp_pytorch_extension_b200.utils import safetensors_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    safetensors_file.save(os.path.join(path, "model.safetensors"), {k: v.to(torch.bfloat16) for k, v in w.items()})


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


TOL = {torch.float32: 2e-4, torch.bfloat16: 6e-2}


def err(got, want):
    """Root mean square of the difference over the last dimension, over that of the wanted values: the worst row."""
    d = (got.detach().cpu().double() - want).pow(2).mean(-1).sqrt()
    return float((d / want.pow(2).mean().sqrt()).max())

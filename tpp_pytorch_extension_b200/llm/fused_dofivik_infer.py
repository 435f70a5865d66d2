"""Dofivik on the hybrid decoder layers: a post-norm decoder whose layers, in any order, are sliding-window latent attention
(with latents of their own or of an earlier layer) or a generalized delta rule, each sub-layer behind a causal input
convolution and with an optional dense xIELU feed-forward.

`DofivikShape.from_config` reads the model's config.json, `load_dofivik` a folder with config.json and model.safetensors,
`build_random_dofivik` draws random weights on the GPU. The runner has the Llama runner's interface: forward, generate
(CUDA-graph decoding), beam_search."""
import json
import os
from dataclasses import dataclass, field

import torch

from .._C import _hybrid_layers as hybrid
from .hybrid_runner import HybridRunner
from .llm_common import get_size


@dataclass
class DofivikShape:
    hidden_size: int
    vocab_size: int
    taps: int
    norm_eps: float
    postln_alpha: float
    layers: list = field(default_factory=list)  # the config's entries: type, mixer, mlp

    @property
    def num_hidden_layers(self):
        return len(self.layers)

    @staticmethod
    def from_config(cfg):
        s = DofivikShape(cfg["width"], cfg["vocab"], cfg["canon"]["taps"], cfg["norm"]["eps"], cfg["postln_alpha"], cfg["layers"])
        for i, l in enumerate(s.layers):
            if l["type"] not in ("latent_attention", "general_delta"):
                raise ValueError(f"layer {i}: unknown mixer type '{l['type']}'")
            if l["mlp"] is not None and l["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind '{l['mlp']['kind']}'")
            if l["type"] == "latent_attention":
                m = l["mixer"]
                if m["rot"]["dims"] != m["rot_dim"]:
                    raise ValueError(f"layer {i}: the rotated part is rotated as a whole (rot.dims = rot_dim)")
                j = m.get("kv_from")
                if j is not None:
                    src = s.layers[j]["mixer"] if 0 <= j < i and s.layers[j]["type"] == "latent_attention" else None
                    if src is None or src.get("kv_from") is not None or (src["kv_rank"], src["rot_dim"]) != (m["kv_rank"], m["rot_dim"]):
                        raise ValueError(f"layer {i}: layer {j} has no latents that it could use")
        return s

    def cache_window(self, i):
        """The longest look-back into layer i's latents, by itself or by a layer that shares them."""
        return max(l["mixer"]["mask"]["size"] for k, l in enumerate(self.layers)
                   if l["type"] == "latent_attention" and (k == i or l["mixer"].get("kv_from") == i))


def make_layer(shape, idx, w, norms, device):
    """w: this layer's tensors under their names without the layer prefix."""
    entry, eps, dtype = shape.layers[idx], shape.norm_eps, norms.dtype
    m = entry["mixer"]
    vec = lambda n: w[n].to(device, torch.float32).contiguous()
    conv = lambda n: w[n].to(device, torch.float32).t().contiguous()  # [taps, D]
    for n in ("canon1", "canon2"):
        if n in w and tuple(w[n].shape) != (shape.hidden_size, shape.taps):
            raise ValueError(f"layer {idx}: {n} has shape {tuple(w[n].shape)}")
    mix = {k[4:]: v for k, v in w.items() if k.startswith("mix.")}
    if entry["type"] == "latent_attention":
        t = {k: mix[k] for k in ("dq", "uq", "uk", "uv", "g", "o")}
        t["dq_norm"] = mix["dq.norm"]
        source = m.get("kv_from")
        if source is None:
            t["dkv"], t["dkv_norm"] = mix["dkv"], mix["dkv.norm"]
        mixer = hybrid.LatentAttention(t, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["mask"]["size"], m["scale"],
                                       m["rot"]["base"], eps, dtype, device, source, shape.cache_window(idx))
    else:
        t = {k: mix[k] for k in ("r", "k", "v", "g", "a", "w1", "w2", "w0", "norm", "o")}
        t["a_bias"] = mix["a.b"]
        mixer = hybrid.GeneralDelta(t, m["heads"], m["dim"], eps, dtype, device)
    if entry["mlp"] is None:
        return hybrid.HybridDecoderLayer(idx, norms, mixer, conv("canon1"), vec("norm1"))
    mlp = hybrid.DenseMlp({"up": w["mlp.up"], "up_bias": w["mlp.up.b"], "down": w["mlp.down"], "down_bias": w["mlp.down.b"],
                           "act_params": w["mlp.act"].float()}, "xielu", dtype, device)
    return hybrid.HybridDecoderLayer(idx, norms, mixer, conv("canon1"), vec("norm1"), mlp, conv("canon2"), vec("norm2"))


class DofivikRunner(HybridRunner):
    def __init__(self, shape, embed, layers, norms, final_w, head_w):
        super().__init__(shape, embed, layers, final_w, head_w, norms.dtype)
        self.norms = norms

    def _embed(self, ids, positions):
        return hybrid.Stream(ids.shape[0], ids.shape[1], ids=ids.contiguous(), embed=self.embed)

    def _head(self, s):
        B, S, _ = s.shape
        return self._logits(self.norms.final(s, self.norm_w, self._wanted_rows(B, S, s.x.device)), B)

    def _stream_rows(self, s, layer, cpp, past):
        return self.norms.enter(s, None, None, cpp.start, None, past)[0]


def _from_tensors(shape, tensors, dtype, device):
    """Runner from name -> tensor; tensors may be a mapping that makes them on demand."""
    if get_size() > 1:
        raise ValueError("this model family runs on one GPU per replica (no tensor-parallel sharding)")
    dev = torch.device(device)
    norms = hybrid.Norms(shape.norm_eps, shape.postln_alpha, dtype)
    layers = []
    for i in range(shape.num_hidden_layers):
        p = f"l{i}."
        layers.append(make_layer(shape, i, {k[len(p):]: tensors[k] for k in tensors if k.startswith(p)}, norms, dev))
    embed = tensors["embed"].to(dev, dtype).contiguous()
    head = hybrid.pad_matrix(tensors["head"].to(dev, dtype), 1, 8)
    if embed.shape != (shape.vocab_size, shape.hidden_size) or head.shape[0] != shape.vocab_size:
        raise ValueError("embedding or head does not have the configured size")
    return DofivikRunner(shape, embed, layers, norms, tensors["final.norm"].to(dev, torch.float32).contiguous(), head)


def load_dofivik(path, dtype=torch.bfloat16, device="cuda"):
    """Model folder -> runner, in bfloat16 or float32."""
    from ..utils import safetensors_file
    with open(os.path.join(path, "config.json")) as f:
        shape = DofivikShape.from_config(json.load(f))
    return _from_tensors(shape, safetensors_file.load(os.path.join(path, "model.safetensors")), dtype, device)


def tensor_shapes(shape, decay_rank=64):
    """Names and shapes of a model's tensors (decay_rank: width of the low-rank decay map, which no config field gives)."""
    D, out = shape.hidden_size, {"embed": (shape.vocab_size, shape.hidden_size)}
    for i, l in enumerate(shape.layers):
        m, p = l["mixer"], f"l{i}."
        H, d = m["heads"], m["dim"]
        out[p + "norm1"], out[p + "canon1"] = (D,), (D, shape.taps)
        if l["type"] == "latent_attention":
            q, r, c, e = m["q_rank"], m["rot_dim"], m["kv_rank"], m["vdim"]
            t = {"dq": (q, D), "dq.norm": (q,), "uq": (H * (d + r), q), "uk": (H * d, c), "uv": (H * e, c), "g": (H, D), "o": (D, H * e)}
            if m.get("kv_from") is None:
                t.update({"dkv": (c + r, D), "dkv.norm": (c,)})
        else:
            t = {n: (H * d, D) for n in "rkvga"}
            t.update({"a.b": (H * d,), "w1": (decay_rank, D), "w2": (H * d, decay_rank), "w0": (H * d,), "norm": (H * d,), "o": (D, H * d)})
        out.update({p + "mix." + k: v for k, v in t.items()})
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            out.update({p + "norm2": (D,), p + "canon2": (D, shape.taps), p + "mlp.up": (F, D), p + "mlp.up.b": (F,), p + "mlp.down": (D, F),
                        p + "mlp.down.b": (D,), p + "mlp.act": (2,)})
    out["final.norm"], out["head"] = (D,), (shape.vocab_size, D)
    return out


def build_random_dofivik(shape, dtype=torch.bfloat16, device="cuda", seed=0, std=0.02, decay_rank=64):
    """Random N(0, std) matrices, norms at one, drawn layer by layer on the device."""
    dev = torch.device(device)
    g = torch.Generator(device=dev).manual_seed(seed)
    shapes = tensor_shapes(shape, decay_rank)

    class Drawn(dict):
        def __getitem__(self, name):
            s = shapes[name]
            if len(s) == 2:
                return (torch.randn(*s, generator=g, device=dev) * std).to(torch.bfloat16)
            plain = name.endswith(("dq.norm", "dkv.norm", "mix.norm"))
            return torch.full(s, 1.0 if plain else 0.0, device=dev)

    return _from_tensors(shape, Drawn.fromkeys(shapes), dtype, device)


def hybrid_shape(layers, hidden, heads, ff, vocab, dim=64, latent_every=4, window=2048, rot_dim=64, kv_rank=512, q_rank=1536, head_dim=128, taps=4):
    """A stack in which every latent_every-th layer is latent attention (every second one sharing the latents of the one
    before it) and the others are delta layers, all with a feed-forward."""
    entries, own = [], None
    for i in range(layers):
        if i % latent_every == latent_every - 1:
            mixer = {"heads": heads, "dim": head_dim, "rot_dim": rot_dim, "vdim": head_dim, "kv_rank": kv_rank, "q_rank": q_rank,
                     "mask": {"size": window}, "scale": (head_dim + rot_dim) ** -0.5, "rot": {"base": 10000.0, "dims": rot_dim}}
            if own is not None:
                mixer["kv_from"], own = own, None
            else:
                own = i
            entries.append({"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff}})
        else:
            entries.append({"type": "general_delta", "mixer": {"heads": hidden // dim, "dim": dim}, "mlp": {"kind": "dense", "ff": ff}})
    return DofivikShape(hidden, vocab, taps, 1e-6, 2.0, entries)


DOFIVIK_8B = hybrid_shape(32, 4096, 32, 14336, 128256)

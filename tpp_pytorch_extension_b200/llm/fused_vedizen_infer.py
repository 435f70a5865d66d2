"""Vedizen on the hybrid decoder layers: parallel layers behind a Dynamic Tanh whose mixers, in any order, are gated linear
attention or chunked differential attention, with an optional clamped gated feed-forward; a range of the layers may be run
several times in a row with the same weights.

`VedizenShape.from_config` reads the model's config.json, `load_vedizen` a folder with config.json and model.safetensors,
`build_random_vedizen` draws random weights on the GPU."""
import json
import os
from dataclasses import dataclass, field

import torch

from .._C import _hybrid_layers as hybrid
from .hybrid_runner import HybridRunner
from .llm_common import get_size

MIXERS = ("gla", "attention")


@dataclass
class VedizenShape:
    hidden_size: int
    vocab_size: int
    norm_eps: float
    embed_scale: float
    layers: list = field(default_factory=list)  # the config's entries: type, mixer, mlp
    loop: tuple = None  # (start, stop, times): layers start .. stop - 1 run `times` times

    @property
    def num_hidden_layers(self):
        return len(self.layers)

    @staticmethod
    def from_config(cfg):
        loop = cfg.get("loop")
        s = VedizenShape(cfg["width"], cfg["vocab"], cfg["norm"]["eps"], cfg["embedding"]["scale"], cfg["layers"],
                         (loop["start"], loop["stop"], loop["times"]) if loop else None)
        for i, l in enumerate(s.layers):
            if l["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type '{l['type']}'")
            if l["mlp"] is not None and l["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind '{l['mlp']['kind']}'")
        if s.loop and not (0 <= s.loop[0] < s.loop[1] <= len(s.layers) and s.loop[2] >= 1):
            raise ValueError(f"the loop over layers {s.loop[0]} .. {s.loop[1] - 1}, {s.loop[2]} times, does not fit {len(s.layers)} layers")
        return s

    def runs(self):
        """(layer, pass of the loop that begins with this run or None), in the order in which the layers run."""
        n = len(self.layers)
        if not self.loop:
            return [(i, None) for i in range(n)]
        start, stop, times = self.loop
        looped = [(i, t if i == start else None) for t in range(times) for i in range(start, stop)]
        return [(i, None) for i in range(start)] + looped + [(i, None) for i in range(stop, n)]


def make_block(shape, idx, w, dtype, device):
    """w: layer idx's tensors under their names without the layer prefix."""
    entry = shape.layers[idx]
    m, mix = entry["mixer"], {k[4:]: v for k, v in w.items() if k.startswith("mix.")}
    if entry["type"] == "gla":
        t = {k: mix[k] for k in ("q", "k", "v", "g", "a1", "a2", "norm", "o")}
        t["a2_bias"] = mix["a2.b"]
        mixer = hybrid.GatedLinearAttention(t, m["heads"], m["dim"], m["vdim"], m["tau"], shape.norm_eps, dtype, device)
    else:
        t = {k: mix[k] for k in ("q", "k", "v", "lq1", "lk1", "lq2", "lk2", "o")}
        t.update({k + "_bias": mix[k + ".b"] for k in ("q", "k", "v")})
        mixer = hybrid.DifferentialAttention(t, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"], m["scale"], m["softcap"], m["diff"],
                                             shape.norm_eps, dtype, device)
    mlp = entry["mlp"]
    return hybrid.ParallelBlock(mixer, None if mlp is None else {k: w["mlp." + k] for k in ("gate", "up", "down")}, None if mlp is None else mlp["limit"],
                                dtype, device)


class VedizenRunner(HybridRunner):
    def __init__(self, shape, embed, layers, first, head_w, dtype):
        super().__init__(shape, embed, layers, None, head_w, dtype)
        self.first = first  # what the first run reads: (vector added in front of it or None, its norm)

    def _embed(self, ids, positions):
        add, norm = self.first
        x, h = hybrid.dynamic_tanh(norm, self.dtype, ids=ids.contiguous(), embed=self.embed, scale=self.shape.embed_scale, add=add)
        return hybrid.NormedStream(ids.shape[0], ids.shape[1], x, h)

    def _head(self, s):
        """The last run's linear has normed the stream for the head already."""
        return self._logits(s.h.index_select(0, self._wanted_rows(s.B, s.S, s.h.device)), s.B)

    def _stream_rows(self, s, layer, cpp, past):
        x = s.x if layer.add is None else s.x - layer.add
        return x[:, :self.shape.hidden_size]


def _from_tensors(shape, tensors, dtype, device):
    """Runner from name -> tensor; tensors may be a mapping that makes them on demand."""
    if get_size() > 1:
        raise ValueError("this model family runs on one GPU per replica (no tensor-parallel sharding)")
    dev = torch.device(device)
    vec = lambda n: hybrid.pad_vector(tensors[n].to(dev, torch.float32)).contiguous()
    norm = lambda n: (float(tensors[n + ".alpha"]), vec(n), vec(n + ".b"))
    blocks, norms = [], []
    for i in range(shape.num_hidden_layers):
        p = f"l{i}."
        blocks.append(make_block(shape, i, {k[len(p):]: tensors[k] for k in tensors if k.startswith(p) and not k.startswith(p + "norm1")}, dtype, dev))
        norms.append(norm(p + "norm1"))
    steps = None
    if shape.loop:
        steps = tensors["loop.step"].to(dev, torch.float32)
        if steps.shape != (shape.loop[2], shape.hidden_size):
            raise ValueError("the loop's step vectors do not have the configured size")
        steps = [hybrid.pad_vector(v).contiguous() for v in steps]
    # in front of every run: the step vector of a pass that begins, and the layer's norm; behind the last one the final norm
    reads = [(None if t is None else steps[t], norms[i]) for i, t in shape.runs()] + [(None, norm("final.norm"))]
    layers = [hybrid.ParallelDecoderLayer(r, blocks[i], *reads[r + 1]) for r, (i, _) in enumerate(shape.runs())]
    embed, head = tensors["embed"].to(dev, dtype), tensors["head"].to(dev, dtype)
    if embed.shape != (shape.vocab_size, shape.hidden_size) or head.shape != embed.shape:
        raise ValueError("embedding or head does not have the configured size")
    return VedizenRunner(shape, hybrid.pad_matrix(embed, 1, 8), layers, reads[0], hybrid.pad_matrix(head, 1, 8), dtype)


def load_vedizen(path, dtype=torch.bfloat16, device="cuda"):
    """Model folder -> runner, in bfloat16 or float32."""
    from ..utils import safetensors_file
    with open(os.path.join(path, "config.json")) as f:
        shape = VedizenShape.from_config(json.load(f))
    return _from_tensors(shape, safetensors_file.load(os.path.join(path, "model.safetensors")), dtype, device)


def tensor_shapes(shape, decay_rank=16):
    """Names and shapes of a model's tensors (decay_rank: width of the low-rank decay map, which no config field gives)."""
    D, out = shape.hidden_size, {"embed": (shape.vocab_size, shape.hidden_size), "head": (shape.vocab_size, shape.hidden_size)}

    def norm(name):
        out.update({name: (D,), name + ".b": (D,), name + ".alpha": ()})

    norm("final.norm")
    if shape.loop:
        out["loop.step"] = (shape.loop[2], D)
    for i, l in enumerate(shape.layers):
        m, p = l["mixer"], f"l{i}."
        H, d, e = m["heads"], m["dim"], m["vdim"]
        norm(p + "norm1")
        if l["type"] == "gla":
            t = {"q": (H * d, D), "k": (H * d, D), "v": (H * e, D), "g": (H * e, D), "a1": (decay_rank, D), "a2": (H * d, decay_rank), "a2.b": (H * d,),
                 "norm": (e,)}
        else:
            G = m["kv_heads"]
            t = {"q": (H * 2 * d, D), "q.b": (H * 2 * d,), "k": (G * 2 * d, D), "k.b": (G * 2 * d,), "v": (G * e, D), "v.b": (G * e,)}
            t.update({n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")})
        t["o"] = (D, H * e)
        out.update({p + "mix." + k: v for k, v in t.items()})
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            out.update({p + "mlp.gate": (F, D), p + "mlp.up": (F, D), p + "mlp.down": (D, F)})
    return out


def build_random_vedizen(shape, dtype=torch.bfloat16, device="cuda", seed=0, std=0.02, decay_rank=16):
    """Random N(0, std) matrices, norms at one, decays near one, drawn layer by layer on the device."""
    dev = torch.device(device)
    g = torch.Generator(device=dev).manual_seed(seed)
    shapes = tensor_shapes(shape, decay_rank)

    class Drawn(dict):
        def __getitem__(self, name):
            s = shapes[name]
            if len(s) == 2:
                return (torch.randn(*s, generator=g, device=dev) * std).to(torch.bfloat16)
            value = 0.5 if name.endswith(".alpha") else 2.0 if name.endswith("a2.b") else 0.0 if name.endswith(".b") else 0.1 if ".mix.l" in name else 1.0
            return torch.full(s, value, device=dev)

    return _from_tensors(shape, Drawn.fromkeys(shapes), dtype, device)


def vedizen_stack(layers, hidden, heads, ff, vocab, attention_every=4, kv_heads=None, chunk=2048, head_dim=64, vdim=128, loop=None):
    """A stack in which every attention_every-th layer is differential attention and the others gated linear attention, all with
    a feed-forward."""
    mlp = {"kind": "dense", "ff": ff, "limit": 7.0}
    attn = {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads or max(1, heads // 4), "dim": head_dim, "vdim": vdim,
                                                        "mask": {"size": chunk}, "scale": head_dim ** -0.5, "softcap": 30.0, "diff": 0.5}}
    gla = {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": head_dim, "vdim": vdim, "tau": 16.0}}
    return VedizenShape(hidden, vocab, 1e-5, 8.0, [attn if i % attention_every == attention_every - 1 else gla for i in range(layers)], loop)


VEDIZEN_8B = vedizen_stack(32, 4096, 32, 14336, 128256)

"""Plain restatement of the Vedizen decoder (parallel sublayers behind a Dynamic Tanh; gated linear attention and chunked
differential attention layers; a run of layers that is passed through several times).

One function per mechanism, written for reading: no batching, no cache, no fusion. It shares no code with the product path
and runs on the CPU in whatever floating-point type the tensors have (the tests use float64). A model is a config
dictionary plus a dictionary of tensors under the names of the checkpoint format."""
import math

import torch


def sigmoid(t):
    return 1.0 / (1.0 + torch.exp(-t))


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def dynamic_tanh(x, w, name):
    """Element by element: no statistics of the vector enter."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def linear(h, w, name):
    y = h @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


# ---------------------------------------------------------------- gated linear attention
def gla_decay(h, w, p, tau):
    """Per token and key channel, in (0, 1)."""
    z = linear(linear(h, w, p + ".a1"), w, p + ".a2")
    return sigmoid(z) ** (1.0 / tau)


def gla_recurrence(q, k, v, a):
    """One head. q, k, a [T, d], v [T, e]; the decay scales the state's rows before the token is written, and the token
    reads what it has written. Returns [T, e]."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.empty_like(v)
    for t in range(q.shape[0]):
        S = a[t].unsqueeze(1) * S + torch.outer(k[t], v[t])
        out[t] = q[t] @ S
    return out


def gla(h, w, p, m, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(h, w, p + ".q").reshape(T, H, d) * d ** -0.5
    k = linear(h, w, p + ".k").reshape(T, H, d)
    v = linear(h, w, p + ".v").reshape(T, H, e)
    a = gla_decay(h, w, p, m["tau"]).reshape(T, H, d)
    o = torch.stack([gla_recurrence(q[:, n], k[:, n], v[:, n], a[:, n]) for n in range(H)], 1)
    o = (over_rms(o, eps) * w[p + ".norm"]).reshape(T, H * e)
    g = linear(h, w, p + ".g")
    return linear(o * g * sigmoid(g), w, p + ".o")


# ---------------------------------------------------------------- differential attention in chunks
def chunk_mask(T, size):
    """[T, T]: token i sees the tokens of its own chunk up to itself."""
    i = torch.arange(T).unsqueeze(1)
    j = torch.arange(T).unsqueeze(0)
    return (j <= i) & (i // size == j // size)


def attention_map(q, k, v, scale, softcap, size):
    """One map of one head: q, k [T, d], v [T, e]."""
    s = softcap * torch.tanh((q @ k.T) * scale / softcap)
    s = s.masked_fill(~chunk_mask(q.shape[0], size), float("-inf"))
    return torch.softmax(s, dim=-1) @ v


def diff_lambda(w, p, diff):
    return torch.exp((w[p + ".lq1"] * w[p + ".lk1"]).sum()) - torch.exp((w[p + ".lq2"] * w[p + ".lk2"]).sum()) + diff


def diff_attention(h, w, p, m, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(h, w, p + ".q").reshape(T, H, 2, d)
    k = linear(h, w, p + ".k").reshape(T, G, 2, d)
    v = linear(h, w, p + ".v").reshape(T, G, e)
    lam = diff_lambda(w, p, m["diff"])
    out = []
    for n in range(H):
        g = n // (H // G)
        a1, a2 = (attention_map(q[:, n, x], k[:, g, x], v[:, g], m["scale"], m["softcap"], m["mask"]["size"]) for x in (0, 1))
        out.append(over_rms(a1 - lam * a2, eps) * (1.0 - m["diff"]))
    return linear(torch.cat(out, -1), w, p + ".o")


# ---------------------------------------------------------------- feed-forward, layers, model
def clamped_glu(h, w, p, limit):
    g = linear(h, w, p + ".gate").clamp(max=limit)
    u = linear(h, w, p + ".up").clamp(-limit, limit)
    return linear(g * sigmoid(1.702 * g) * (u + 1.0), w, p + ".down")


def layer(x, w, i, entry, eps):
    h = dynamic_tanh(x, w, f"l{i}.norm1")
    mixer = {"gla": gla, "attention": diff_attention}[entry["type"]]
    y = mixer(h, w, f"l{i}.mix", entry["mixer"], eps)
    if entry["mlp"] is not None:
        y = y + clamped_glu(h, w, f"l{i}.mlp", entry["mlp"]["limit"])
    return x + y


def layer_runs(cfg):
    """(layer, pass or None if no step vector comes right before it) in the order in which the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence from its first token; layers_out (a list) receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, t in layer_runs(cfg):
        if t is not None:
            x = x + w["loop.step"][t]
        x = layer(x, w, i, cfg["layers"][i], eps)
        if layers_out is not None:
            layers_out.append(x)
    return linear(dynamic_tanh(x, w, "final.norm"), w, "head")


def random_model(cfg, seed=0, gain=1.0, rank=5):
    """Random tensors for a config (float64, values representable in bfloat16). gain scales queries and keys, so that
    attention scores stand out from one another; rank is the width of the low-rank decay map."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    w = {}

    def put(name, *shape, std=None, mean=0.0):
        std = std if std is not None else shape[-1] ** -0.5
        w[name] = (torch.randn(shape, generator=g, dtype=torch.float64) * std + mean).to(torch.bfloat16).to(torch.float64)

    def norm(name):
        put(name, D, std=0.2, mean=1.0)
        put(name + ".b", D, std=0.2)
        put(name + ".alpha", std=0.05, mean=0.5)

    put("embed", V, D, std=1.0 / cfg["embedding"]["scale"])
    put("head", V, D)
    norm("final.norm")
    if cfg.get("loop"):
        put("loop.step", cfg["loop"]["times"], D, std=0.5)
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix."
        norm(f"l{i}.norm1")
        H, d, e = m["heads"], m["dim"], m["vdim"]
        if l["type"] == "gla":
            put(p + "q", H * d, D, std=2 * D ** -0.5)
            put(p + "k", H * d, D)
            put(p + "v", H * e, D)
            put(p + "g", H * e, D)
            put(p + "a1", rank, D)
            put(p + "a2", H * d, rank, std=1.0)
            put(p + "a2.b", H * d, std=1.0, mean=1.0)
            put(p + "norm", e, std=0.2, mean=1.0)
        else:
            G = m["kv_heads"]
            put(p + "q", H * 2 * d, D, std=gain * D ** -0.5)
            put(p + "q.b", H * 2 * d, std=0.3)
            put(p + "k", G * 2 * d, D, std=gain * D ** -0.5)
            put(p + "k.b", G * 2 * d, std=0.3)
            put(p + "v", G * e, D)
            put(p + "v.b", G * e, std=0.3)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                put(p + n, d, std=0.1)
        put(p + "o", D, H * e)
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            put(f"l{i}.mlp.gate", F, D, std=1.5 * D ** -0.5)
            put(f"l{i}.mlp.up", F, D, std=1.5 * D ** -0.5)
            put(f"l{i}.mlp.down", D, F)
    return w

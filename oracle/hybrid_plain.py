"""Plain restatement of the Dofivik decoder (post-norm hybrid of latent attention and generalized-delta layers).

One function per mechanism, written for reading: token by token or key by key, no batching, no cache, no fusion. It
shares no code with the product path and runs on the CPU in whatever floating-point type the tensors have (the tests use
float64). A model is a config dictionary plus a dictionary of tensors under the names of the checkpoint format."""
import math

import torch


def softplus(t):
    return torch.log1p(torch.exp(-t.abs())) + t.clamp(min=0)


def sigmoid(t):
    return 1.0 / (1.0 + torch.exp(-t))


def rms(x, eps):
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    """The model's norm: the weight is stored as its distance from one."""
    return rms(x, eps) * (1.0 + w)


def causal_conv(h, w):
    """Per-channel convolution over time. h [T, D], w [D, taps]; the last tap meets the current token."""
    T, taps = h.shape[0], w.shape[1]
    out = torch.zeros_like(h)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def rotate_pairs(x, positions, base):
    """Rotary embedding of neighbouring pairs. x [T, ..., dims], positions [T]."""
    dims = x.shape[-1]
    out = torch.empty_like(x)
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        ang = (positions.to(torch.float64) * f).reshape(-1, *([1] * (x.dim() - 2)))
        c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_attention(q, k, v, scale, window):
    """q, k [T, H, d], v [T, H, e]: token i sees tokens j with 0 <= i - j < window."""
    T = q.shape[0]
    i = torch.arange(T).unsqueeze(1)
    j = torch.arange(T).unsqueeze(0)
    seen = (i - j >= 0) & (i - j < window)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~seen, float("-inf"))
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, dim=-1), v)


def latent_of(w, p, m, h, eps):
    """The two things a latent-attention layer caches: the normed latent and the rotated key part."""
    both = h @ w[p + ".mix.dkv"].T
    c = rms(both[:, :m["kv_rank"]], eps) * w[p + ".mix.dkv.norm"]
    k_rot = rotate_pairs(both[:, m["kv_rank"]:], torch.arange(h.shape[0]), m["rot"]["base"])
    return c, k_rot


def latent_attention(w, p, m, h, latent, eps):
    """Mixer on its own (already convolved) input h [T, D]; latent = latent_of(...) of this or of the shared layer."""
    T, H, d, r, e = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_rot = latent
    cq = rms(h @ w[p + ".mix.dq"].T, eps) * w[p + ".mix.dq.norm"]
    q = (cq @ w[p + ".mix.uq"].T).reshape(T, H, d + r)
    q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], torch.arange(T), m["rot"]["base"])], -1)
    k = (c @ w[p + ".mix.uk"].T).reshape(T, H, d)
    k = torch.cat([k, k_rot.unsqueeze(1).expand(T, H, r)], -1)
    v = (c @ w[p + ".mix.uv"].T).reshape(T, H, e)
    o = window_attention(q, k, v, m["scale"], m["mask"]["size"])
    o = o * sigmoid(h @ w[p + ".mix.g"].T).unsqueeze(-1)
    return o.reshape(T, H * e) @ w[p + ".mix.o"].T


def delta_step(S, r, k, v, decay, rate):
    """One token of one head. S [dim, dim] (key channel, value channel); returns the new state and the read-out."""
    u = k / torch.sqrt((k * k).sum() + 1e-6)
    S = decay.unsqueeze(1) * S - torch.outer(rate * u, u @ S) + torch.outer(k, v)
    return S, r @ S


def general_delta(w, p, m, h, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    r = (h @ w[p + ".mix.r"].T).reshape(T, H, d)
    k = (h @ w[p + ".mix.k"].T).reshape(T, H, d)
    v = (h @ w[p + ".mix.v"].T).reshape(T, H, d)
    lora = torch.tanh(h @ w[p + ".mix.w1"].T) @ w[p + ".mix.w2"].T + w[p + ".mix.w0"]
    decay = torch.exp(-math.exp(-0.5) * sigmoid(lora)).reshape(T, H, d)
    rate = sigmoid(h @ w[p + ".mix.a"].T + w[p + ".mix.a.b"]).reshape(T, H, d)
    out = torch.empty(T, H, d, dtype=h.dtype)
    for n in range(H):
        S = torch.zeros(d, d, dtype=h.dtype)
        for t in range(T):
            S, out[t, n] = delta_step(S, r[t, n], k[t, n], v[t, n], decay[t, n], rate[t, n])
    out = rms(out, eps).reshape(T, H * d) * w[p + ".mix.norm"]
    return (out * sigmoid(h @ w[p + ".mix.g"].T)) @ w[p + ".mix.o"].T


def xielu(z, a):
    pos = softplus(a[0]) * z * z + 0.5 * z
    neg = (0.5 + softplus(a[1])) * (torch.exp(z.clamp(max=0)) - 1.0 - z) + 0.5 * z
    return torch.where(z > 0, pos, neg)


def dense_mlp(w, p, h):
    z = h @ w[p + ".mlp.up"].T + w[p + ".mlp.up.b"]
    return xielu(z, w[p + ".mlp.act"]) @ w[p + ".mlp.down"].T + w[p + ".mlp.down.b"]


def forward(cfg, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence from its first token; layers_out (a list) receives the stream after every layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.as_tensor(tokens)]
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        h = x + causal_conv(x, w[p + ".canon1"])
        if layer["type"] == "latent_attention":
            j = m.get("kv_from")
            if j is None:
                latents[i] = latent_of(w, p, m, h, eps)
                j = i
            y = latent_attention(w, p, m, h, latents[j], eps)
        elif layer["type"] == "general_delta":
            y = general_delta(w, p, m, h, eps)
        else:
            raise ValueError(layer["type"])
        x = zero_centred_norm(alpha * x + y, w[p + ".norm1"], eps)
        if layer["mlp"] is not None:
            h = x + causal_conv(x, w[p + ".canon2"])
            x = zero_centred_norm(alpha * x + dense_mlp(w, p, h), w[p + ".norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return zero_centred_norm(x, w["final.norm"], eps) @ w["head"].T


def random_model(cfg, seed=0, gain=1.0):
    """Random tensors for a config (float64, values representable in bfloat16). gain scales the projections that make
    queries and latents, so that attention scores stand out from one another. Low-rank width of the decay: cfg key
    'decay_rank' of the mixer (default 8)."""
    g = torch.Generator().manual_seed(seed)
    D, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    w = {}

    def put(name, *shape, std=None, mean=0.0):
        std = std if std is not None else shape[-1] ** -0.5
        w[name] = (torch.randn(*shape, generator=g, dtype=torch.float64) * std + mean).to(torch.bfloat16).to(torch.float64)

    put("embed", V, D, std=1.0)
    put("head", V, D)
    put("final.norm", D, std=0.2)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        put(p + ".norm1", D, std=0.2)
        put(p + ".canon1", D, taps, std=0.3)
        H, d = m["heads"], m["dim"]
        if layer["type"] == "latent_attention":
            q, r, c, e = m["q_rank"], m["rot_dim"], m["kv_rank"], m["vdim"]
            put(p + ".mix.dq", q, D)
            put(p + ".mix.dq.norm", q, std=0.2, mean=1.0)
            put(p + ".mix.uq", H * (d + r), q, std=gain * q ** -0.5)
            if m.get("kv_from") is None:
                put(p + ".mix.dkv", c + r, D)
                put(p + ".mix.dkv.norm", c, std=0.2, mean=1.0)
            put(p + ".mix.uk", H * d, c, std=gain * c ** -0.5)
            put(p + ".mix.uv", H * e, c)
            put(p + ".mix.g", H, D)
            put(p + ".mix.o", D, H * e)
        else:
            k = m.get("decay_rank", 8)
            for n in "rkvga":
                put(f"{p}.mix.{n}", H * d, D)
            put(p + ".mix.a.b", H * d, std=0.5)
            put(p + ".mix.w1", k, D)
            put(p + ".mix.w2", H * d, k)
            put(p + ".mix.w0", H * d, std=0.5, mean=-2.0)
            put(p + ".mix.norm", H * d, std=0.2, mean=1.0)
            put(p + ".mix.o", D, H * d)
        if layer["mlp"] is not None:
            put(p + ".norm2", D, std=0.2)
            put(p + ".canon2", D, taps, std=0.3)
            F = layer["mlp"]["ff"]
            put(p + ".mlp.up", F, D)
            put(p + ".mlp.up.b", F, std=0.2)
            put(p + ".mlp.down", D, F)
            put(p + ".mlp.down.b", D, std=0.2)
            put(p + ".mlp.act", 2, std=0.5)
    return w

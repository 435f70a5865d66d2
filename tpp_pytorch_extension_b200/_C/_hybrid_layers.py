"""Layers of hybrid decoders on the kernels of include/tpx_hybrid.h: latent attention with a sliding window, the
generalized delta rule and a dense feed-forward, each behind a post-norm residual with an input convolution; gated linear
attention and chunked differential attention beside a clamped gated feed-forward in parallel layers.

Activations are bf16 or, for a model built in float32, true 32-bit throughout; the residual stream, norms, gates, angles,
scores and recurrent states are 32-bit in both. Weight matrices are stored with their rows padded to whole 16-byte units
(zeros), activations likewise, so that every size reaches the same kernels."""
import ctypes

import torch

from .. import _lib
from .. import _timers
from ._fused_llm_infer import bf16_linear_scratch

ACT = {None: 0, "gelu": 1, "silu": 2, "relu": 3, "tanh": 4, "xielu": 5, "clamped_glu": 6}


def round_up(n, m):
    return (n + m - 1) // m * m


def pad_matrix(w, rows=8, cols=8):
    """w [N, K] with zero rows / columns up to multiples of `rows` / `cols`."""
    N, K = w.shape
    return torch.nn.functional.pad(w, (0, round_up(K, cols) - K, 0, round_up(N, rows) - N)).contiguous()


def pad_vector(v, m=8):
    return torch.nn.functional.pad(v, (0, round_up(v.numel(), m) - v.numel())).contiguous()


def _call(name, st):
    rc = getattr(_lib.lib(), name)(ctypes.byref(st), _lib.stream())
    if rc:
        _lib.check(rc)


def _linear_call(x, w, y, bias=None, **fields):
    M, (N, K) = x.shape[0], w.shape
    if x.dtype != w.dtype or x.shape[1] != K:
        raise _lib.TpxError(f"linear: input {tuple(x.shape)} {x.dtype} does not fit the weight {tuple(w.shape)} {w.dtype}")
    sc = _lib.scratch(bf16_linear_scratch(M), x.device)
    _call("tpx_linear", _lib.LinearStruct(
        w=w.data_ptr(), x=x.data_ptr(), bias=_lib.ptr(bias), y=_lib.ptr(y), M=M, N=N, K=K, ldw=w.stride(0), ldx=x.stride(0),
        ldy=y.stride(0) if y is not None else 0, f32=int(w.dtype == torch.float32), out_f32=int(y is not None and y.dtype == torch.float32),
        scratch=sc.data_ptr(), scratch_bytes=sc.numel(), **fields))


def linear(x, w, bias=None, act=None, act_from=0, act_params=None, out_f32=False):
    """act(x . w^T + bias): x [M, >= K] and w [N, K] of one type (bf16 or fp32), rows possibly strided; bias and act_params
    fp32; the activation applies to output columns from act_from on. Result bf16 unless the operands are fp32 or out_f32."""
    y = torch.empty((x.shape[0], w.shape[0]), dtype=torch.float32 if (w.dtype == torch.float32 or out_f32) else torch.bfloat16, device=x.device)
    _linear_call(x, w, y, bias, act=ACT[act], act_from=act_from, act_params=_lib.ptr(act_params))
    return y


def linear_glu(x, w, bias, act_from, limit, z):
    """x . w^T + bias whose columns from act_from on are (gate, up) pairs of clamped gated units: these go to z [M, units]
    (rows possibly strided), the columns before them are returned."""
    y = torch.empty((x.shape[0], act_from), dtype=w.dtype, device=x.device)
    _linear_call(x, w, y, bias, act=ACT["clamped_glu"], act_from=act_from, limit=limit, z=z.data_ptr(), ldz=z.stride(0))
    return y


def linear_residual(x, w, res, add, norm):
    """The residual stream behind a linear and the norm of its next reader, norm = (alpha, w, b): x_out = res + x . w^T + add
    (fp32 [M, N]; add may be None) and tanh(alpha x_out) w + b in the type of x."""
    alpha, nw, nb = norm
    x_out, h = torch.empty_like(res), torch.empty(res.shape, dtype=x.dtype, device=x.device)
    _linear_call(x, w, None, res=res.data_ptr(), add=_lib.ptr(add), norm_w=nw.data_ptr(), norm_b=nb.data_ptr(), norm_alpha=alpha,
                 x_out=x_out.data_ptr(), h=h.data_ptr(), ldr=res.stride(0), ldh=h.stride(0))
    return x_out, h


def argmax_rows_f32(x):
    """Greedy pick over the last dimension of fp32 logits [..., n] -> int64 [...]."""
    x = x.contiguous()
    n = x.shape[-1]
    out = torch.empty(x.shape[:-1], dtype=torch.int64, device=x.device)
    _lib.check(_lib.lib().tpx_argmax_f32(x.data_ptr(), x.numel() // n, n, out.data_ptr(), _lib.stream()))
    return out


class Stream:
    """The residual stream between two sub-layers: either token ids that have not been embedded yet, or x and the last
    sub-layer's output y, whose sum with x (and norm w) the next sub-layer's first kernel takes. All fp32."""

    def __init__(self, B, S, ids=None, embed=None, x=None, y=None, w=None):
        self.B, self.S, self.ids, self.embed, self.x, self.y, self.w = B, S, ids, embed, x, y, w

    @property
    def shape(self):
        return (self.B, self.S, (self.embed if self.ids is not None else self.x).shape[-1])


class Norms:
    """Constants of the residual path shared by all layers of a model."""

    def __init__(self, eps, alpha, dtype):
        self.eps, self.alpha, self.dtype = float(eps), float(alpha), dtype

    def enter(self, s, conv, state, start, dev_len, past):
        """Close the pending sub-layer and open the next: returns (x [T, D] fp32, h [T, D padded])."""
        B, S, D = s.shape
        dev = (s.ids if s.ids is not None else s.x).device
        x = torch.empty((B * S, D), dtype=torch.float32, device=dev)
        h, taps = None, 0
        if conv is not None:
            taps = conv.shape[0]
            h = torch.empty((B * S, round_up(D, 8)), dtype=self.dtype, device=dev)
        _call("tpx_postnorm_conv", _lib.PostnormConvStruct(
            ids=_lib.ptr(s.ids), embed=_lib.ptr(s.embed) if s.ids is not None else None, x=_lib.ptr(s.x), y=_lib.ptr(s.y), w=_lib.ptr(s.w),
            conv=_lib.ptr(conv), state=_lib.ptr(state), start=_lib.ptr(start), dev_len=_lib.ptr(dev_len), x_out=x.data_ptr(), h=_lib.ptr(h),
            B=B, S=S, D=D, ldh=h.shape[1] if h is not None else 0, past=past, alpha=self.alpha, eps=self.eps, taps=taps,
            f32=int(self.dtype == torch.float32)))
        return x, h

    def final(self, s, w_final, rows):
        """Final norm of the token rows `rows` (int64 indices)."""
        D = s.shape[2]
        out = torch.empty((rows.numel(), round_up(D, 8)), dtype=self.dtype, device=rows.device)
        _call("tpx_postnorm_final", _lib.PostnormFinalStruct(
            x=s.x.data_ptr(), y=s.y.data_ptr(), w=s.w.data_ptr(), w_final=w_final.data_ptr(), rows=rows.data_ptr(), out=out.data_ptr(),
            n=rows.numel(), D=D, ldo=out.shape[1], alpha=self.alpha, eps=self.eps, f32=int(self.dtype == torch.float32)))
        return out


class Step:
    """What the layers of one call share: sequences, new and cached token counts, padding."""

    def __init__(self, B, S, past, start, dev_len):
        self.B, self.S, self.past, self.start, self.dev_len = B, S, past, start, dev_len


class LatentAttention:
    """Attention over a cached latent (and one rotated key part shared by all heads) in a sliding window.

    weights: dq [q_rank, D], dq_norm, uq [heads * (dim + rot_dim), q_rank], uk [heads * dim, kv_rank], uv [heads * vdim,
    kv_rank], g [heads, D], o [D, heads * vdim] and, unless the latents of another layer are used (`source`, that layer's
    index), dkv [kv_rank + rot_dim, D], dkv_norm. cache_window: the longest look-back of this layer's latents by any layer."""

    def __init__(self, w, heads, dim, rot_dim, vdim, kv_rank, window, scale, rot_base, eps, dtype, device, source=None, cache_window=None):
        self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank = heads, dim, rot_dim, vdim, kv_rank
        self.window, self.scale, self.eps, self.source, self.dtype = min(int(window), 1 << 29), float(scale), float(eps), source, dtype
        self.cache_window = min(int(cache_window or window), 1 << 29)
        mat = lambda t: t.to(device, dtype)
        vec = lambda t: t.to(device, torch.float32).contiguous()
        self.q_rank = w["dq"].shape[0]
        self.krp = round_up(kv_rank, 16)
        self.R = self.krp + round_up(rot_dim, 16) + 8  # 16 mod 32 bytes: the rows of a page start in different banks
        down = [w["dq"]] + ([w["dkv"]] if source is None else []) + [w["g"]]
        self.down = pad_matrix(mat(torch.cat(down, 0)))
        self.q_norm = vec(w["dq_norm"])
        self.kv_norm = vec(w["dkv_norm"]) if source is None else None
        self.uq = pad_matrix(mat(w["uq"]))
        self.uk = pad_matrix(mat(w["uk"]), 1, 16)
        self.uv = pad_matrix(mat(w["uv"]), 1, 16)
        # keys and values of a multi-token call as one linear of the latents, where its kernel serves the head sizes
        self.kv = None
        if dtype == torch.bfloat16 and _lib.lib().tpx_latent_prefill_serves(dim, rot_dim, vdim):
            self.kv = pad_matrix(torch.cat([self.uk, self.uv], 0))
            self.uk, self.uv = self.kv[:heads * dim], self.kv[heads * dim:heads * (dim + vdim)]
        self.o = pad_matrix(mat(w["o"]), 1, 8)
        half = torch.arange(rot_dim // 2, dtype=torch.float64)
        self.freq = (float(rot_base) ** (-2.0 * half / max(rot_dim, 1))).to(device)

    def reserve(self, lc, B, tokens, device):
        if self.source is None:
            lc.ensure_latent(B, self.R, tokens, self.cache_window, self.dtype, device)

    def forward(self, h, lc, cache, step):
        B, S, past, T, f32 = step.B, step.S, step.past, step.B * step.S, int(self.dtype == torch.float32)
        dev = h.device
        src = lc if self.source is None else cache.layers[self.source]
        proj = linear(h, self.down, out_f32=True)
        cq = torch.empty((T, self.uq.shape[1]), dtype=self.dtype, device=dev)
        cos_sin = torch.empty((T, max(self.rot_dim // 2, 1), 2), dtype=torch.float32, device=dev)
        gate = torch.empty((T, self.heads), dtype=torch.float32, device=dev)
        lat, L = None, 0
        if self.source is None:
            if step.dev_len is None:
                lc.ensure_latent(B, self.R, S, self.cache_window, self.dtype, dev)
            if S > 1:  # several tokens: their rows, behind those of the cached tokens still in reach, in one piece
                back = min(past, self.cache_window - 1)
                L = back + S
                lat = torch.empty((B, L, self.R), dtype=self.dtype, device=dev)
                if back:
                    _lib.check(_lib.lib().tpx_latent_gather(lc.ptrs.data_ptr(), lc.pages(), B, self.R, past, back, L, lat.data_ptr(), f32, _lib.stream()))
                lc.live = lat
        elif S > 1:
            lat = src.live
            L = lat.shape[1]
        _call("tpx_latent_prep", _lib.LatentPrepStruct(
            proj=proj.data_ptr(), q_norm=self.q_norm.data_ptr(), kv_norm=_lib.ptr(self.kv_norm), freq=_lib.ptr(self.freq), start=_lib.ptr(step.start),
            dev_len=_lib.ptr(step.dev_len), cq=cq.data_ptr(), cos_sin=cos_sin.data_ptr(), gate=gate.data_ptr(), lat=_lib.ptr(lat),
            pages=src.ptrs.data_ptr(), B=B, S=S, L=L, ldp=proj.shape[1], ldq=cq.shape[1], past=past, npages=src.pages(), q_rank=self.q_rank,
            kv_rank=self.kv_rank, krp=self.krp, rot_dim=self.rot_dim, R=self.R, heads=self.heads, eps=self.eps, own_kv=int(self.source is None), f32=f32))
        q = linear(cq, self.uq)
        out = torch.empty((T, self.o.shape[1]), dtype=self.dtype, device=dev)
        if S > 1 and self.kv is not None:
            kv = linear(lat.view(B * L, self.R)[:, :self.krp], self.kv)
            _call("tpx_latent_prefill", _lib.LatentPrefillStruct(
                q=q.data_ptr(), kv=kv.data_ptr(), lat=lat.data_ptr(), cos_sin=cos_sin.data_ptr(), gate=gate.data_ptr(), start=_lib.ptr(step.start),
                out=out.data_ptr(), B=B, S=S, L=L, past=past, heads=self.heads, dim=self.dim, rot_dim=self.rot_dim, vdim=self.vdim, krp=self.krp, R=self.R,
                ldq=q.shape[1], ldkv=kv.shape[1], ldo=out.shape[1], window=self.window, scale=self.scale))
            return linear(out, self.o, out_f32=True)
        qa = torch.empty((T, self.heads, self.R), dtype=self.dtype, device=dev)
        _call("tpx_latent_absorb", _lib.LatentAbsorbStruct(
            q=q.data_ptr(), w_uk=self.uk.data_ptr(), cos_sin=cos_sin.data_ptr(), qa=qa.data_ptr(), T=T, ldq=q.shape[1], heads=self.heads, dim=self.dim,
            kv_rank=self.kv_rank, krp=self.krp, rot_dim=self.rot_dim, R=self.R, f32=f32))
        ol = torch.empty((T, self.heads, self.krp), dtype=self.dtype, device=dev)
        _call("tpx_latent_attn", _lib.LatentAttnStruct(
            qa=qa.data_ptr(), lat=_lib.ptr(lat), pages=src.ptrs.data_ptr(), start=_lib.ptr(step.start), dev_len=_lib.ptr(step.dev_len), ol=ol.data_ptr(),
            B=B, S=S, L=L, past=past, npages=src.pages(), heads=self.heads, krp=self.krp, R=self.R, window=self.window, scale=self.scale, f32=f32))
        _call("tpx_latent_value", _lib.LatentValueStruct(
            ol=ol.data_ptr(), gate=gate.data_ptr(), w_uv=self.uv.data_ptr(), out=out.data_ptr(), T=T, heads=self.heads, vdim=self.vdim, krp=self.krp,
            ldo=out.shape[1], f32=f32))
        return linear(out, self.o, out_f32=True)


class GeneralDelta:
    """Generalized delta rule with a decay per key channel from a low-rank map.

    weights: r, k, v, g, a [heads * dim, D], a_bias, w1 [rank, D], w2 [heads * dim, rank], w0, norm [heads * dim],
    o [D, heads * dim]."""

    def __init__(self, w, heads, dim, eps, dtype, device):
        self.heads, self.dim, self.eps, self.dtype = heads, dim, float(eps), dtype
        mat = lambda t: t.to(device, dtype)
        vec = lambda t: t.to(device, torch.float32).contiguous()
        hd = heads * dim
        five = pad_matrix(mat(torch.cat([w[n] for n in ("r", "k", "v", "a", "g")], 0)))
        self.low = five.shape[0]  # first column of the low-rank part, on a 16-byte boundary
        self.proj = torch.cat([five, pad_matrix(mat(w["w1"]))], 0).contiguous()
        self.w2 = pad_matrix(mat(w["w2"]), 1, 8)
        self.w0, self.a_bias, self.norm = vec(w["w0"]), vec(w["a_bias"]), vec(w["norm"])
        self.o = pad_matrix(mat(w["o"]), 1, 8)
        assert self.w0.numel() == hd and self.o.shape[1] == round_up(hd, 8)

    def state(self, lc, B, device):
        return lc.state("delta", (B, self.heads, self.dim, self.dim), device)

    def reserve(self, lc, B, tokens, device):
        self.state(lc, B, device)

    def forward(self, h, lc, cache, step):
        B, S, T, f32 = step.B, step.S, step.B * step.S, int(self.dtype == torch.float32)
        dev, hd = h.device, self.heads * self.dim
        proj = linear(h, self.proj, act="tanh", act_from=self.low)
        wraw = linear(proj[:, self.low:], self.w2, bias=self.w0, out_f32=True)
        state = self.state(lc, B, dev)
        raw = torch.empty((T, hd), dtype=torch.float32, device=dev)
        out = torch.empty((T, self.o.shape[1]), dtype=self.dtype, device=dev)
        _call("tpx_delta_rule", _lib.DeltaRuleStruct(
            proj=proj.data_ptr(), wraw=wraw.data_ptr(), a_bias=self.a_bias.data_ptr(), norm_w=self.norm.data_ptr(), start=_lib.ptr(step.start),
            dev_len=_lib.ptr(step.dev_len), state=state.data_ptr(), raw=raw.data_ptr(), out=out.data_ptr(), B=B, S=S, past=step.past, ldp=proj.shape[1],
            ldo=out.shape[1], heads=self.heads, dim=self.dim, eps=self.eps, f32=f32))
        return linear(out, self.o, out_f32=True)


class DenseMlp:
    """down(act(up h + b)) + b. weights: up [F, D], up_bias, down [D, F], down_bias; act "xielu" takes the two numbers
    act_params = (p, q)."""

    def __init__(self, w, act, dtype, device):
        mat = lambda t: t.to(device, dtype)
        self.act, self.act_params = act, None
        if act == "xielu":
            sp = torch.nn.functional.softplus(w["act_params"].double(), threshold=1e9)
            self.act_params = torch.stack([sp[0], 0.5 + sp[1]]).to(device, torch.float32).contiguous()
        self.up, self.down = pad_matrix(mat(w["up"])), pad_matrix(mat(w["down"]), 1, 8)
        self.up_bias = pad_vector(w["up_bias"].to(device, torch.float32))
        self.down_bias = w["down_bias"].to(device, torch.float32).contiguous()

    def forward(self, h):
        z = linear(h, self.up, bias=self.up_bias, act=self.act, act_params=self.act_params)
        return linear(z, self.down, bias=self.down_bias, out_f32=True)


class HybridDecoderLayer:
    """x <- norm1(alpha x + mixer(x + conv1(x))); with a feed-forward also x <- norm2(alpha x + mlp(x + conv2(x))).

    The norm that closes a sub-layer runs in the kernel that opens the next one, so forward takes and returns a Stream."""

    def __init__(self, idx, norms, mixer, conv1, norm1, mlp=None, conv2=None, norm2=None):
        self.idx, self.norms, self.mixer, self.mlp = idx, norms, mixer, mlp
        self.conv1, self.norm1, self.conv2, self.norm2 = conv1, norm1, conv2, norm2

    def _conv_state(self, lc, name, conv, B, device):
        taps, D = conv.shape
        return lc.state(name, (B, taps - 1, D), device)

    def reserve(self, cache, B, tokens, device):
        """Cache storage for B sequences of up to `tokens` tokens."""
        lc = cache.hybrid_layer(self.idx)
        self.mixer.reserve(lc, B, tokens, device)
        self._conv_state(lc, "conv1", self.conv1, B, device)
        if self.mlp is not None:
            self._conv_state(lc, "conv2", self.conv2, B, device)

    def forward(self, inp, cache, use_cache=True, dev_len=None):
        """inp = [Stream, start int32 [B] or None, ...]: the interface of the other decoder layers."""
        s, start = inp[0], inp[1]
        B, S, D = s.shape
        lc = cache.hybrid_layer(self.idx)
        dev = (s.ids if s.ids is not None else s.x).device
        past = lc.offset
        step = Step(B, S, past, start, dev_len)
        sc = _timers.scope
        st1 = self._conv_state(lc, "conv1", self.conv1, B, dev)
        with sc("norm_conv", 0, 0):
            x, h = self.norms.enter(s, self.conv1, st1, start, dev_len, past)
        with sc("mixer", 0, 0):
            y = self.mixer.forward(h, lc, cache, step)
        s = Stream(B, S, x=x, y=y, w=self.norm1)
        if self.mlp is not None:
            st2 = self._conv_state(lc, "conv2", self.conv2, B, dev)
            with sc("norm_conv", 0, 0):
                x, h = self.norms.enter(s, self.conv2, st2, start, dev_len, past)
            with sc("mlp", 0, 0):
                y = self.mlp.forward(h)
            s = Stream(B, S, x=x, y=y, w=self.norm2)
        if dev_len is None:
            lc.offset += S
        return [s]


def dynamic_tanh(norm, dtype, ids=None, embed=None, scale=1.0, x=None, add=None):
    """The stream at its start, scale embed[ids], or a given x [n, D], plus add; returns (stream fp32, its norm in `dtype`)."""
    alpha, w, b = norm
    src = ids if ids is not None else x
    n, D = (ids.numel(), embed.shape[1]) if ids is not None else x.shape
    x_out, h = torch.empty((n, D), dtype=torch.float32, device=src.device), torch.empty((n, round_up(D, 8)), dtype=dtype, device=src.device)
    _call("tpx_dyt", _lib.DytStruct(ids=_lib.ptr(ids), embed=_lib.ptr(embed) if ids is not None else None, x=_lib.ptr(x), add=_lib.ptr(add), w=w.data_ptr(),
                                    b=b.data_ptr(), x_out=x_out.data_ptr(), h=h.data_ptr(), n=n, D=D, ldh=h.shape[1], scale=scale, alpha=alpha,
                                    f32=int(dtype == torch.float32)))
    return x_out, h


def _sections(parts):
    """Row blocks of one linear, each padded to whole 16-byte units: (their rows stacked, first row of each)."""
    at, cols = 0, []
    for p in parts:
        cols.append(at)
        at += round_up(p.shape[0], 8)
    return torch.cat([pad_matrix(p) for p in parts], 0), cols


class GatedLinearAttention:
    """Linear attention with a decay per key channel from a low-rank map.

    weights: q, k [heads * dim, D], v, g [heads * vdim, D], a1 [rank, D], a2 [heads * dim, rank], a2_bias, norm [vdim],
    o [D, heads * vdim]. The projections are rows `self.rows` of the layer's input linear."""

    def __init__(self, w, heads, dim, vdim, tau, eps, dtype, device):
        self.heads, self.dim, self.vdim, self.tau, self.eps, self.dtype = heads, dim, vdim, float(tau), float(eps), dtype
        mat = lambda t: t.to(device, dtype)
        vec = lambda t: t.to(device, torch.float32).contiguous()
        for n, rows in (("q", dim), ("k", dim), ("v", vdim), ("g", vdim), ("a2", dim)):
            if w[n].shape[0] != heads * rows:
                raise ValueError(f"gated linear attention: '{n}' has {w[n].shape[0]} rows, {heads} heads of {rows} are configured")
        self.rows, self.cols = _sections([mat(w[n]) for n in ("q", "k", "v", "g", "a1")])
        self.rows_bias = None
        self.rank = w["a1"].shape[0]
        self.a2, self.a2_bias, self.norm = pad_matrix(mat(w["a2"]), 1, 8), vec(w["a2_bias"]), vec(w["norm"])
        self.o = pad_matrix(mat(w["o"]), 1, 8)
        self.fused_decay = bool(_lib.lib().tpx_gla_token_serves(dim, vdim))

    def state(self, lc, B, device):
        return lc.state("gla", (B, self.heads, self.dim, self.vdim), device)

    def reserve(self, lc, B, tokens, device):
        self.state(lc, B, device)

    def forward(self, proj, out, lc, cache, step):
        """proj [T, >= rows]: the input linear's result; out [T, heads * vdim]: columns of the output linear's input."""
        B, S, T = step.B, step.S, step.B * step.S
        dev, (q, k, v, g, a1) = proj.device, self.cols
        zraw = raw = None
        if S > 1 or not self.fused_decay:
            zraw = linear(proj[:, a1:a1 + self.a2.shape[1]], self.a2, bias=self.a2_bias, out_f32=True)
            raw = torch.empty((T, self.heads * self.vdim), dtype=torch.float32, device=dev)
        _call("tpx_gla", _lib.GlaStruct(
            proj=proj.data_ptr(), zraw=_lib.ptr(zraw), a2=self.a2.data_ptr(), a2_bias=self.a2_bias.data_ptr(), norm_w=self.norm.data_ptr(),
            start=_lib.ptr(step.start), dev_len=_lib.ptr(step.dev_len), state=self.state(lc, B, dev).data_ptr(), raw=_lib.ptr(raw), out=out.data_ptr(),
            B=B, S=S, past=step.past, ldp=proj.stride(0), ldo=out.stride(0), lda2=self.a2.stride(0), rank=self.rank, heads=self.heads, dim=self.dim,
            vdim=self.vdim, q_col=q, k_col=k, v_col=v, g_col=g, a1_col=a1, tau=self.tau, eps=self.eps, f32=int(self.dtype == torch.float32)))


class DifferentialAttention:
    """Differential attention (two maps per head over shared values) with capped scores, within chunks of the sequence.

    weights: q [heads * 2 * dim, D], k [kv_heads * 2 * dim, D], v [kv_heads * vdim, D] and their biases q_bias, k_bias, v_bias,
    lq1, lk1, lq2, lk2 [dim], o [D, heads * vdim]. diff: the constant part of lambda."""

    def __init__(self, w, heads, kv_heads, dim, vdim, chunk, scale, softcap, diff, eps, dtype, device):
        self.heads, self.kv_heads, self.dim, self.vdim, self.eps, self.dtype = heads, kv_heads, dim, vdim, float(eps), dtype
        self.chunk, self.scale, self.softcap = min(int(chunk), 1 << 29), float(scale), float(softcap)
        mat = lambda t: t.to(device, dtype)
        if heads % kv_heads:
            raise ValueError(f"differential attention: {heads} heads cannot share {kv_heads} key/value heads evenly")
        for n, rows in (("q", heads * 2 * dim), ("k", kv_heads * 2 * dim), ("v", kv_heads * vdim)):
            if w[n].shape[0] != rows:
                raise ValueError(f"differential attention: '{n}' has {w[n].shape[0]} rows, {rows} are configured")
        self.rows, self.cols = _sections([mat(w[n]) for n in ("q", "k", "v")])
        self.rows_bias = torch.cat([pad_vector(w[n + "_bias"].to(device, torch.float32)) for n in ("q", "k", "v")])
        l = {n: w[n].double() for n in ("lq1", "lk1", "lq2", "lk2")}
        self.lam = float(torch.exp((l["lq1"] * l["lk1"]).sum()) - torch.exp((l["lq2"] * l["lk2"]).sum()) + diff)
        self.mult = 1.0 - float(diff)
        self.o = pad_matrix(mat(w["o"]), 1, 8)
        self.R = 2 * round_up(dim, 16) + round_up(vdim, 16) + 8  # both keys, the value; 16 mod 32 bytes: rows start in different banks
        self.direct = dtype == torch.bfloat16 and bool(_lib.lib().tpx_diff_prefill_serves(dim, vdim, self.softcap))

    def reserve(self, lc, B, tokens, device):
        lc.ensure_pages((B, self.kv_heads, 32, self.R), tokens, self.chunk, self.dtype, device)

    def forward(self, proj, out, lc, cache, step):
        B, S, past = step.B, step.S, step.past
        dev, (q, k, v) = proj.device, self.cols
        if step.dev_len is None:
            self.reserve(lc, B, S, dev)
        live, L = None, S
        if S > 1:  # the cached tokens still in reach come in front of the call's own
            L += min(past, self.chunk - 1)
            if L > S or not self.direct:
                live = torch.empty((B, L, self.kv_heads, self.R), dtype=self.dtype, device=dev)
        _call("tpx_diff_attn", _lib.DiffAttnStruct(
            proj=proj.data_ptr(), pages=lc.ptrs.data_ptr(), live=_lib.ptr(live), start=_lib.ptr(step.start), dev_len=_lib.ptr(step.dev_len),
            out=out.data_ptr(), B=B, S=S, L=L, past=past, npages=lc.pages(), ldp=proj.stride(0), ldo=out.stride(0), heads=self.heads,
            kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, R=self.R, chunk=self.chunk, q_col=q, k_col=k, v_col=v, scale=self.scale,
            softcap=self.softcap, lam=self.lam, mult=self.mult, eps=self.eps, f32=int(self.dtype == torch.float32)))


class NormedStream:
    """The residual stream between two parallel layers: x [T, D] fp32 and h, its norm for the next reader."""

    def __init__(self, B, S, x, h):
        self.B, self.S, self.x, self.h = B, S, x, h

    @property
    def shape(self):
        return (self.B, self.S, self.x.shape[-1])


class ParallelBlock:
    """Weights of a layer whose mixer and feed-forward read one normed input and are added together: one linear for everything
    that reads it, with the gated units made in its epilogue, and one for both outputs, [o | down] on the columns
    [mixer | units]. mlp: None or a dict with gate, up [F, D], down [D, F]; limit: its clamp."""

    def __init__(self, mixer, mlp, limit, dtype, device):
        self.mixer, self.limit = mixer, float(limit) if mlp is not None else 0.0
        mat = lambda t: t.to(device, dtype)
        rows, bias, cols = [mixer.rows], mixer.rows_bias, [mixer.o]
        self.act_from, self.units = mixer.rows.shape[0], 0
        if mlp is not None:
            gate, up = pad_matrix(mat(mlp["gate"])), pad_matrix(mat(mlp["up"]))
            self.units = gate.shape[0]
            rows.append(torch.stack([gate, up], 1).reshape(2 * self.units, -1))
            cols.append(pad_matrix(mat(mlp["down"]), 1, 8))
            if bias is not None:
                bias = torch.nn.functional.pad(bias, (0, 2 * self.units))
        self.w_in, self.bias_in = torch.cat(rows, 0).contiguous(), bias
        self.w_out = pad_matrix(torch.cat(cols, 1), 8, 1)
        mixer.rows = None  # part of w_in now
        self.mixer_cols = mixer.o.shape[1]
        self.padded = self.mixer_cols != mixer.heads * mixer.vdim
        mixer.o = None

    def forward(self, s, lc, cache, step, add, norm):
        T, dev = step.B * step.S, s.h.device
        sc = _timers.scope
        cat = (torch.zeros if self.padded else torch.empty)((T, self.mixer_cols + self.units), dtype=s.h.dtype, device=dev)
        with sc("parallel_in", 0, 0):
            if self.units:
                proj = linear_glu(s.h, self.w_in, self.bias_in, self.act_from, self.limit, cat[:, self.mixer_cols:])
            else:
                proj = linear(s.h, self.w_in, self.bias_in)
        with sc("mixer", 0, 0):
            self.mixer.forward(proj, cat, lc, cache, step)
        with sc("parallel_out", 0, 0):
            x, h = linear_residual(cat, self.w_out, s.x, add, norm)
        return NormedStream(step.B, step.S, x, h)


class ParallelDecoderLayer:
    """x <- x + (mixer(h) + mlp(h)), h the norm of x. One run of a block: several runs may share a block (a looped stack of
    layers), each with the cache `idx` of its own. add, norm: the vector that comes onto the stream behind this run (or None)
    and the norm (alpha, w, b) of what reads it next."""

    def __init__(self, idx, block, add, norm):
        self.idx, self.block, self.add, self.norm = idx, block, add, norm

    def reserve(self, cache, B, tokens, device):
        self.block.mixer.reserve(cache.hybrid_layer(self.idx), B, tokens, device)

    def forward(self, inp, cache, use_cache=True, dev_len=None):
        """inp = [NormedStream, start int32 [B] or None, ...]: the interface of the other decoder layers."""
        s, start = inp[0], inp[1]
        lc = cache.hybrid_layer(self.idx)
        s = self.block.forward(s, lc, cache, Step(s.B, s.S, lc.offset, start, dev_len), self.add, self.norm)
        if dev_len is None:
            lc.offset += s.S
        return [s]

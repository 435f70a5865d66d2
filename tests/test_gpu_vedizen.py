"""The Vedizen decoder's kernels, cache and runner against the plain implementation of oracle/vedizen_plain.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

from oracle import vedizen_plain as P
from tests import vedizen_util as U
from tests.test_gpu_hybrid import CUTS, DTYPES, portions

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
HALF = {torch.float32: 2e-5, torch.bfloat16: 1.5e-2}  # one linear, one rounding; a row may be a single large value


def rnd(seed, *shape, std=1.0):
    """Normal values that bf16 holds exactly."""
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64) * std).to(torch.bfloat16).double()


# ---------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,D", [(1, 8), (7, 96), (33, 520)])
def test_dynamic_tanh(cuda, dtype, n, D):
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    w = {"n": rnd(1, D), "n.b": rnd(2, D), "n.alpha": torch.tensor(0.8).double()}
    norm = (0.8, w["n"].float().to(cuda), w["n.b"].float().to(cuda))
    embed, ids, add = rnd(3, 11, D), torch.arange(n) * 3 % 11, rnd(4, D)
    for a in (None, add):
        x = embed[ids] * 2.5 + (0 if a is None else a)
        gx, gh = HL.dynamic_tanh(norm, dtype, ids=ids.to(cuda), embed=embed.to(cuda, dtype), scale=2.5, add=None if a is None else a.float().to(cuda))
        assert U.err(gx, x) < 1e-6 and U.err(gh, P.dynamic_tanh(x, w, "n")) < HALF[dtype]
        gx, gh = HL.dynamic_tanh(norm, dtype, x=embed[ids].float().to(cuda), add=None if a is None else a.float().to(cuda))
        x = embed[ids] + (0 if a is None else a)
        assert U.err(gx, x) < 1e-6 and U.err(gh, P.dynamic_tanh(x, w, "n")) < HALF[dtype]


SHAPES = [(1, 136, 8), (5, 200, 72), (16, 96, 264), (17, 264, 128), (40, 96, 2048), (70, 128, 64), (130, 264, 320), (300, 72, 136), (2, 512, 4096)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", SHAPES)
def test_linear_with_gated_units(cuda, dtype, M, N, K):
    """Columns before act_from as they are, the rest as clamped gated units; act_from inside, at the edge and across tiles."""
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    x, w, b = rnd(M, M, K + 8), rnd(N, N, K, std=2 * K ** -0.5), rnd(K, N)
    xd = x.to(cuda, dtype)[:, 8:]
    y = x[:, 8:] @ w.T + b
    for act_from in (8, N // 16 * 8, N - 2):
        g, u = y[:, act_from::2], y[:, act_from + 1::2]
        z = g.clamp(max=1.3)
        z = z * P.sigmoid(1.702 * z) * (u.clamp(-1.3, 1.3) + 1)
        buf = torch.full((M, z.shape[1] + 24), 7.0, dtype=dtype, device=cuda)
        got = HL.linear_glu(xd, w.to(cuda, dtype), b.float().to(cuda), act_from, 1.3, buf[:, 16:])
        assert got.shape == (M, act_from) and U.err(got, y[:, :act_from]) < HALF[dtype]
        assert U.err(buf[:, 16:16 + z.shape[1]], z) < HALF[dtype]
        assert (buf[:, :16] == 7).all() and (buf[:, 16 + z.shape[1]:] == 7).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", SHAPES)
def test_linear_into_the_stream(cuda, dtype, M, N, K):
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    x, w, res, add = rnd(M, M, K), rnd(N, N, K, std=K ** -0.5), rnd(3, M, N), rnd(4, N)
    n = {"n": rnd(1, N), "n.b": rnd(2, N), "n.alpha": torch.tensor(0.6).double()}
    norm = (0.6, n["n"].float().to(cuda), n["n.b"].float().to(cuda))
    for a in (None, add):
        want = res + x @ w.T + (0 if a is None else a)
        gx, gh = HL.linear_residual(x.to(cuda, dtype), w.to(cuda, dtype), res.float().to(cuda), None if a is None else a.float().to(cuda), norm)
        assert gx.dtype == torch.float32 and U.err(gx, want) < 5e-6  # the sum stays 32-bit in both types
        assert gh.dtype == dtype and U.err(gh, P.dynamic_tanh(want, n, "n")) < HALF[dtype]


def mixer_of(cfg, w, i, cuda, dtype):
    """Layer i's mixer, with its part of the input linear and of the output linear."""
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    from tpp_pytorch_extension_b200.llm import fused_vedizen_infer as FV
    shape, kept = FV.VedizenShape.from_config(cfg), {}

    class Keep:
        def __init__(self, mixer, *a):
            kept["mixer"] = mixer
    real, HL.ParallelBlock = HL.ParallelBlock, Keep
    try:
        FV.make_block(shape, i, {k[3:]: v.float() for k, v in w.items() if k.startswith(f"l{i}.")}, dtype, cuda)
    finally:
        HL.ParallelBlock = real
    return kept["mixer"]


def mixer_over(m, h, cut, cuda, dtype, start=None, cache=None):
    """Mixer over h [B, T, D] in portions; [B, T, D]. start: leading padding per sequence."""
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    from tpp_pytorch_extension_b200._C._tpp_attn import TppCache
    cache = cache or TppCache()
    B, T, D = h.shape
    lc, outs, t = cache.hybrid_layer(0), [], 0
    st = torch.tensor([0] * B if start is None else start, dtype=torch.int32, device=cuda)
    hd = torch.nn.functional.pad(h.float(), (0, -D % 8)).to(cuda, dtype)
    for n in portions(T, cut):
        proj = HL.linear(hd[:, t:t + n].reshape(B * n, -1).contiguous(), m.rows, m.rows_bias)
        out = torch.zeros((B * n, m.o.shape[1] + 16), dtype=dtype, device=cuda)
        m.forward(proj, out, lc, cache, HL.Step(B, n, t, st, None))
        assert not out[:, m.o.shape[1]:].any()
        lc.offset += n
        outs.append(HL.linear(out[:, :m.o.shape[1]], m.o, out_f32=True).view(B, n, D))
        t += n
    return torch.cat(outs, 1)


def plain_batch(f, h, start):
    """f over every sequence of h [B, T, D] without its padding; padding rows are zero."""
    want = torch.zeros_like(h)
    for b, n in enumerate(start):
        want[b, n:] = f(h[b, n:])
    return want


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,tau", [(2, 8, 8, 1.0), (3, 20, 28, 8.0), (1, 32, 64, 16.0), (2, 48, 72, 16.0), (4, 64, 40, 4.0), (2, 96, 128, 16.0), (2, 128, 256, 16.0),
                                                (1, 160, 24, 2.0), (1, 300, 7, 16.0), (1, 5, 300, 3.0), (2, 24, 320, 16.0)])
def test_gla_alone(cuda, dtype, heads, dim, vdim, tau):
    cfg = U.config([U.gla(heads, dim, vdim, tau, mlp=None)])
    w = P.random_model(cfg, seed=dim, rank=11)
    T = 70 if dim <= 128 else 40
    h = rnd(dim, T, cfg["width"])
    want = P.gla(h, w, "l0.mix", cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
    m = mixer_of(cfg, w, 0, cuda, dtype)
    for cut in CUTS:
        assert U.err(mixer_over(m, h[None], cut, cuda, dtype)[0], want) < U.TOL[dtype], cut


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,vdim", [(16, 64), (32, 128), (24, 200), (64, 64), (56, 128), (64, 256), (128, 40), (128, 128), (96, 256)])
def test_gla_many_heads(cuda, dtype, dim, vdim):
    """Enough (sequence, head) pairs for whole heads per block; unequal padding, portions of several sizes."""
    B, H, T, start = 50, 6, 23, [(7 * b) % 11 for b in range(50)]
    cfg = U.config([U.gla(H, dim, vdim, mlp=None)], width=48)
    w = P.random_model(cfg, seed=dim + vdim)
    h = rnd(1, B, T, 48)
    some = [0, 1, 17, 49]
    f = lambda x: P.gla(x, w, "l0.mix", cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
    want = plain_batch(f, h[some], [start[b] for b in some])
    m = mixer_of(cfg, w, 0, cuda, dtype)
    for cut in ([10 ** 6], [2], [9, 1], [16, 5]):
        got = mixer_over(m, h, cut, cuda, dtype, start)
        assert U.err(got[some].reshape(-1, 48), want.reshape(-1, 48)) < U.TOL[dtype], cut
        assert torch.isfinite(got).all()


@pytest.mark.parametrize("shift,tau", [(8.0, 16.0), (-60.0, 1.0), (-300.0, 0.5), (0.0, 0.05)])
def test_gla_decays_at_their_ends(cuda, shift, tau):
    """Decays close to one over a long sequence (what was written far back stays) and decays that vanish within a token."""
    for heads, dim, vdim, B in ((2, 64, 64, 1), (1, 128, 128, 1), (3, 40, 24, 1), (6, 32, 64, 50)):
        cfg = U.config([U.gla(heads, dim, vdim, tau, mlp=None)], width=48)
        w = P.random_model(cfg, seed=1)
        w["l0.mix.a2.b"] = torch.where(torch.arange(heads * dim) % 3 == 0, shift, 2.0).double()
        h = rnd(3, 1, 500 if B == 1 else 40, 48)
        want = P.gla(h[0], w, "l0.mix", cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
        for dtype in DTYPES:
            m = mixer_of(cfg, w, 0, cuda, dtype)
            for cut in ([10 ** 6], [480, 1], [37]):
                got = mixer_over(m, h.expand(B, -1, -1), cut, cuda, dtype)
                assert U.err(got[-1], want) < U.TOL[dtype], (heads, dtype, cut)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [1, 2, 31, 32, 33, 64, 65, 128, 129, 1000])
def test_diff_attention_alone(cuda, dtype, chunk):
    """High gain so that single keys dominate and an edge that is one token off shows."""
    cfg = U.config([U.attn(chunk=chunk, mlp=None)])
    w = P.random_model(cfg, seed=chunk, gain=4.0)
    T = 300
    h = rnd(1, T, cfg["width"])
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    want = P.diff_attention(h, w, "l0.mix", m, eps)
    off = P.diff_attention(h, w, "l0.mix", dict(m, mask={"size": chunk + 1}), eps)
    assert chunk == 1000 or U.err(off, want) > 4 * U.TOL[dtype]
    mix = mixer_of(cfg, w, 0, cuda, dtype)
    for cut in CUTS + [[130, 7], [257, 1]]:
        assert U.err(mixer_over(mix, h[None], cut, cuda, dtype)[0], want) < U.TOL[dtype], cut


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [dict(heads=8, kv_heads=2, dim=64, vdim=128), dict(heads=1, kv_heads=1, dim=1, vdim=1), dict(heads=16, kv_heads=1, dim=40, vdim=24),
                                   dict(heads=6, kv_heads=3, dim=128, vdim=64), dict(heads=18, kv_heads=2, dim=16, vdim=32), dict(heads=4, kv_heads=4, dim=96, vdim=104),
                                   dict(heads=2, kv_heads=1, dim=136, vdim=200), dict(heads=3, kv_heads=3, dim=128, vdim=128), dict(heads=2, kv_heads=2, dim=10, vdim=18)])
def test_diff_attention_sizes(cuda, dtype, sizes):
    if sizes["vdim"] == 1 and dtype == torch.bfloat16:
        pytest.skip("a norm over one value leaves its sign only, which rounding turns over where the maps cancel")
    cfg = U.config([U.attn(chunk=150, scale=sizes["dim"] ** -0.5, mlp=None, **sizes)])
    w = P.random_model(cfg, seed=3, gain=2.0)
    B, T, start = 2, 260, [0, 19]
    h = rnd(1, B, T, cfg["width"])
    want = plain_batch(lambda x: P.diff_attention(x, w, "l0.mix", cfg["layers"][0]["mixer"], cfg["norm"]["eps"]), h, start)
    mix = mixer_of(cfg, w, 0, cuda, dtype)
    for cut in ([10 ** 6], [165, 1], [90, 60, 2]):
        got = mixer_over(mix, h, cut, cuda, dtype, start)
        assert U.err(got.reshape(B * T, -1), want.reshape(B * T, -1)) < U.TOL[dtype], cut


@pytest.mark.parametrize("dim,vdim,B,chunk", [(64, 128, 40, 700), (128, 128, 2, 610), (32, 40, 3, 2000)])
def test_diff_attention_long_chunks(cuda, dim, vdim, B, chunk):
    """Many tiles per query tile and many pages per warp, with enough sequences that one block takes a whole chunk; unequal
    padding moves the chunks against the pages."""
    cfg = U.config([U.attn(8, 4, dim, vdim, chunk, dim ** -0.5, 20.0, mlp=None)], width=64)
    w = P.random_model(cfg, seed=3, gain=3.0)
    T, start = 900, [(31 * b) % 170 for b in range(B)]
    h = rnd(1, B, T, 64)
    some = sorted({0, 1, B - 1})
    want = plain_batch(lambda x: P.diff_attention(x, w, "l0.mix", cfg["layers"][0]["mixer"], cfg["norm"]["eps"]), h[some], [start[b] for b in some])
    mix = mixer_of(cfg, w, 0, cuda, torch.bfloat16)
    for cut in ([10 ** 6], [600, 299, 1], [869, 1]):
        got = mixer_over(mix, h, cut, cuda, torch.bfloat16, start)[some]
        assert U.err(got.reshape(-1, 64), want.reshape(-1, 64)) < U.TOL[torch.bfloat16], cut


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("softcap,gain", [(0.5, 3.0), (2.0, 3.0), (64.0, 3.0), (64.0, 30.0), (200.0, 3.0)])
def test_scores_far_above_and_below_the_cap(cuda, dtype, softcap, gain):
    cfg = U.config([U.attn(4, 2, 32, 32, 90, 0.2, softcap, mlp=None)])
    w = P.random_model(cfg, seed=5, gain=gain)
    if gain > 10:  # scores of hundreds: make queries and keys small integers, exact in bf16, as a rounded score would be amplified
        for n in ("q", "k"):
            w[f"l0.mix.{n}"] = torch.zeros_like(w[f"l0.mix.{n}"])
            w[f"l0.mix.{n}"][:, :4] = rnd(9, w[f"l0.mix.{n}"].shape[0], 4).mul(2).round()
            w[f"l0.mix.{n}.b"] *= 0
    h = rnd(2, 150, cfg["width"])
    h[:, :4] = h[:, :4].round()
    want = P.diff_attention(h, w, "l0.mix", cfg["layers"][0]["mixer"], cfg["norm"]["eps"])
    mix = mixer_of(cfg, w, 0, cuda, dtype)
    for cut in ([10 ** 6], [100, 1], [95, 2]):
        assert U.err(mixer_over(mix, h[None], cut, cuda, dtype)[0], want) < U.TOL[dtype], cut


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk", [45, 64, 200])
def test_diff_attention_single_far_key(cuda, dtype, chunk):
    """One key of map 1 stands out by far: all later tokens of its chunk return its value, the next chunk's first does not.
    The key is a chunk's first token, one in the middle, or its last."""
    cfg = U.config([U.attn(2, 1, 16, 24, chunk, 1.0, 30.0, mlp=None)])
    w = P.random_model(cfg, seed=5)
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    w["l0.mix.q"] *= 0
    w["l0.mix.k"] *= 0
    w["l0.mix.k.b"] *= 0
    w["l0.mix.q.b"] = rnd(6, 64).sign()
    w["l0.mix.k"][:16, 0] = w["l0.mix.q.b"][:16]  # map 1 of head 0: the score is 16 times the input's first channel
    T = 2 * chunk + 40
    for at in (chunk, chunk + 17, 2 * chunk - 1):
        h = rnd(7, T, cfg["width"])
        h[:, 0] = 0
        h[at, 0] = 1.5
        want = P.diff_attention(h, w, "l0.mix", m, eps)
        edge = min(2 * chunk, T - 1)
        for size in (chunk - 1, chunk + 1):
            assert U.err(P.diff_attention(h, w, "l0.mix", dict(m, mask={"size": size}), eps)[chunk:], want[chunk:]) > 0.3
        mix = mixer_of(cfg, w, 0, cuda, dtype)
        for cut in ([10 ** 6], [at + 1, 1], [2 * chunk, 1], [chunk + 5, 2]):
            got = mixer_over(mix, h[None], cut, cuda, dtype)[0]
            for t in sorted({at, min(at + 1, T - 1), edge - 1, edge, T - 1}):
                assert U.err(got[t:t + 1], want[t:t + 1]) < 2 * U.TOL[dtype], (at, cut, t)


# ---------------------------------------------------------------- whole models
def run_portions(r, toks, cut, cuda):
    cache, outs, t = None, [], 0
    r.only_last_logit = False
    for n in portions(len(toks), cut):
        lg, cache = r.forward(torch.tensor([toks[t:t + n]], device=cuda), None, None, cache)
        outs.append(lg[0])
        t += n
    return torch.cat(outs, 0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_model_layers_and_portions(cuda, dtype, name):
    cfg, w = U.model(name)
    r = U.runner_of(cfg, w, dtype)
    toks = U.tokens(cfg, 140 if name != "wide" else 120)
    layers = []
    want = P.forward(cfg, w, toks, layers)
    r.layer_outputs = []
    assert U.err(run_portions(r, toks, CUTS[0], cuda), want) < U.TOL[dtype]
    assert len(r.layer_outputs) == len(layers)
    for got, lw in zip(r.layer_outputs, layers):
        assert U.err(got, lw) < U.TOL[dtype]
    r.layer_outputs = None
    for cut in CUTS[1:]:
        assert U.err(run_portions(r, toks, cut, cuda), want) < U.TOL[dtype], cut


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_unequal_batch_against_each_alone(cuda, dtype, name):
    cfg, w = U.model(name, seed=4)
    r = U.runner_of(cfg, w, dtype)
    lens, steps = [1, 50, 2, 33, 97], 40
    seqs = [U.tokens(cfg, n + steps, seed=i) for i, n in enumerate(lens)]
    want = [P.forward(cfg, w, s) for s in seqs]
    width = max(lens)
    ids = torch.tensor([[0] * (width - n) + s[:n] for n, s in zip(lens, seqs)], device=cuda)
    mask = torch.tensor([[0] * (width - n) + [1] * n for n in lens], device=cuda)
    r.only_last_logit = True
    lg, cache = r.forward(ids, mask)
    alive = list(range(len(lens)))
    for t in range(steps):
        for row, i in enumerate(alive):
            assert U.err(lg[row], want[i][lens[i] + t - 1:lens[i] + t]) < U.TOL[dtype], (i, t)
        if t in (5, 20):  # some sequences end; the others go on in a smaller batch
            gone = 0 if t == 5 else 1
            alive.pop(gone)
            cache.get_cpp().keep_sequences([k for k in range(len(alive) + 1) if k != gone])
        ids = torch.tensor([[seqs[i][lens[i] + t]] for i in alive], device=cuda)
        lg, cache = r.forward(ids, None, None, cache)


@pytest.mark.parametrize("dtype", DTYPES)
def test_what_else_is_in_the_batch_changes_nothing(cuda, dtype):
    """The same sequence alone, beside others, with other padding: equal up to rounding, also against itself in bf16."""
    cfg, w = U.model("mixed", seed=12)
    r = U.runner_of(cfg, w, dtype)
    r.only_last_logit = False
    a, b = U.tokens(cfg, 70, 1), U.tokens(cfg, 90, 2)
    alone = run_portions(r, a, [10 ** 6], cuda)
    ids = torch.tensor([[0] * 20 + a, b, b[:40] + a[:50]], device=cuda)
    lg, _ = r.forward(ids, torch.tensor([[0] * 20 + [1] * 70, [1] * 90, [1] * 90], device=cuda))
    assert U.err(lg[0, 20:], alone.cpu().double()) < (1e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("dtype,name", [(torch.float32, "mixed"), (torch.bfloat16, "mixed"), (torch.bfloat16, "wide")])
def test_storage_used_again(cuda, dtype, name):
    """A cache whose pages and states held another request gives what a fresh one gives, also when the pages hold NaN."""
    cfg, w = U.model(name, seed=6)
    r = U.runner_of(cfg, w, dtype)
    r.only_last_logit = False
    a, b = U.tokens(cfg, 150, 1), U.tokens(cfg, 90, 2)
    want = P.forward(cfg, w, b)
    _, cache = r.forward(torch.tensor([a], device=cuda))
    for poison in (False, True):
        cache.get_cpp().reset()
        if poison:
            for lc in cache.get_cpp().layers:
                for t in lc.arenas:
                    t.fill_(float("nan"))
        lg, _ = r.forward(torch.tensor([b[:40]], device=cuda), None, None, cache)
        got = [lg[0]]
        lg, _ = r.forward(torch.tensor([b[40:47]], device=cuda), None, None, cache)
        got.append(lg[0])
        for t in range(47, 90):
            lg, _ = r.forward(torch.tensor([[b[t]]], device=cuda), None, None, cache)
            got.append(lg[0])
        assert U.err(torch.cat(got, 0), want) < U.TOL[dtype]


def greedy(cfg, w, prompt, n):
    t, margins = list(prompt), []
    for _ in range(n):
        top = P.forward(cfg, w, t)[-1].topk(2)
        margins.append(float(top.values[0] - top.values[1]))
        t.append(int(top.indices[0]))
    return t, margins


def test_greedy_generation(cuda):
    """generate() (graph-replayed and eager, padded batch, reused session) against greedy decoding with the plain model."""
    cfg, w = U.model("odd", seed=9)
    r = U.runner_of(cfg, w, torch.float32)
    lens, new = [3, 11, 7], 24
    prompts = [U.tokens(cfg, n, seed=20 + i) for i, n in enumerate(lens)]
    want = [greedy(cfg, w, p, new) for p in prompts]

    def check(prompts, want, **kw):
        width = max(len(p) for p in prompts)
        ids = torch.tensor([[0] * (width - len(p)) + p for p in prompts], device=cuda)
        mask = torch.tensor([[0] * (width - len(p)) + [1] * len(p) for p in prompts], device=cuda)
        out = r.generate(ids, new, attention_mask=mask, **kw).cpu()
        for i, (t, margins) in enumerate(want):
            got = out[i, width - len(prompts[i]):].tolist()
            for k in range(len(t)):
                if k >= len(prompts[i]) and margins[k - len(prompts[i])] < 1e-3:
                    break  # a tie: either token is right, and what follows differs
                assert got[k] == t[k], (i, k)

    check(prompts, want)
    assert r._session is not None and r._session.graph is not None
    graph = r._session.graph
    check(prompts, want)                       # replays the recorded step in the same cache
    assert r._session.graph is graph
    other = [U.tokens(cfg, n, seed=40 + i) for i, n in enumerate([5, 4, 9])]
    check(other, [greedy(cfg, w, p, new) for p in other])
    assert r._session.graph is graph
    check(prompts, want, use_graph=False)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_passes_many_chunks(cuda, dtype):
    """Decoding through several chunks in the recorded step: every token is the plain model's choice behind the tokens so far."""
    cfg, w = U.model(U.config([U.attn(chunk=33), U.gla(2, 32, 40), U.attn(chunk=64, dim=32, vdim=32), U.attn(chunk=5, mlp=None)], loop=(1, 3, 2)), seed=2, gain=2.0)
    r = U.runner_of(cfg, w, dtype)
    prompt, new = U.tokens(cfg, 6), 300
    out = r.generate(torch.tensor([prompt], device=cuda), new)[0].cpu().tolist()
    assert all(lc.pages() <= lc.window_pages() for lc in r._session.cache.get_cpp().layers if lc.arenas)
    lg = P.forward(cfg, w, out)
    margin = 1e-3 if dtype == torch.float32 else 0.25 * float(lg.std())
    sure = 0
    for t in range(len(prompt) - 1, len(out) - 1):
        top = lg[t].topk(2)
        if float(top.values[0] - top.values[1]) > margin:
            sure += 1
            assert out[t + 1] == int(top.indices[0]), t
    assert sure > 50


def test_beam_search_scores(cuda):
    cfg, w = U.model("one", seed=3)
    r = U.runner_of(cfg, w, torch.float32)
    ids = torch.tensor([U.tokens(cfg, 9, 1), U.tokens(cfg, 9, 2)], device=cuda)
    seqs, scores = r.beam_search(ids, 6, num_beams=3)
    for b in range(2):
        for k in range(3):
            t = seqs[b, k].tolist()
            lp = torch.log_softmax(P.forward(cfg, w, t), -1)
            want = sum(float(lp[i, t[i + 1]]) for i in range(8, 14))
            assert abs(want - float(scores[b, k])) < 1e-3 * max(1.0, abs(want))


def test_looped_runs_have_caches_of_their_own(cuda):
    cfg, w = U.model("mixed")
    r = U.runner_of(cfg, w, torch.float32)
    _, cache = r.forward(torch.tensor([U.tokens(cfg, 20)], device=cuda))
    layers = cache.get_cpp().layers
    assert len(layers) == len(r.layers) == 1 + 3 * 3 + 1 and len({id(l.block) for l in r.layers}) == 5
    assert len({a.data_ptr() for lc in layers for a in lc.arenas + list(lc.states.values())}) == len(layers)


def test_bad_input_is_refused(cuda):
    from tpp_pytorch_extension_b200 import _lib
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    cfg, w = U.model("one")
    r = U.runner_of(cfg, w, torch.float32)
    with pytest.raises(ValueError):
        r.forward(torch.tensor([[cfg["vocab"]]], device=cuda))
    _, cache = r.forward(torch.tensor([[1, 2]], device=cuda))
    with pytest.raises(ValueError):
        r.forward(torch.tensor([[1], [2]], device=cuda), None, None, cache)
    with pytest.raises(Exception):
        cache.crop(1)
    x = torch.zeros(2, 16, device=cuda)
    with pytest.raises(_lib.TpxError):
        HL.linear_glu(x, torch.zeros(8, 16, device=cuda), None, 3, 1.0, x)  # an odd first column
    with pytest.raises(_lib.TpxError):
        HL.linear(x, torch.zeros(8, 12, device=cuda))
    with pytest.raises(_lib.TpxError):
        HL._call("tpx_gla", _lib.GlaStruct(B=1, S=1, heads=1, dim=600, vdim=8, tau=1.0))
    with pytest.raises(_lib.TpxError):
        HL._call("tpx_diff_attn", _lib.DiffAttnStruct(B=1, S=1, L=1, heads=3, kv_heads=2, dim=8, vdim=8, chunk=4, npages=1, softcap=1.0))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_command(cuda, tmp_path, dtype):
    """bin/trace_run on a saved folder: a prompt, a batch of unequal prompts that ends one by one, and single tokens."""
    cfg, w = U.model("mixed", seed=8)
    U.save_folder(tmp_path / "m", cfg, w)
    (tmp_path / "o").mkdir()
    a, b, c = U.tokens(cfg, 60, 1), U.tokens(cfg, 45, 2), U.tokens(cfg, 5, 3)
    steps = [{"step": 0, "entries": [{"id": "c", "tokens": c, "want": [0, 4]}], "end": ["c"]},
             {"step": 1, "entries": [{"id": "a", "tokens": a[:50], "want": [49]}, {"id": "b", "tokens": b[:40], "want": [3, 39]}], "end": []}]
    for i in range(10):
        e = [{"id": "a", "tokens": [a[50 + i]], "want": [0]}]
        if i < 5:
            e.insert(0, {"id": "b", "tokens": [b[40 + i]], "want": [0] if i % 2 else []})
        steps.append({"step": 2 + i, "entries": e, "end": ["b"] if i == 4 else ["a"] if i == 9 else []})
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path / "o")],
                       input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    ref = {"a": P.forward(cfg, w, a), "b": P.forward(cfg, w, b), "c": P.forward(cfg, w, c)}
    at = {"a": 0, "b": 0, "c": 0}
    for s in steps:
        want = []
        for e in s["entries"]:
            want += [ref[e["id"]][at[e["id"]] + k] for k in e["want"]]
            at[e["id"]] += len(e["tokens"])
        f = tmp_path / "o" / f"{s['step']}.f32"
        assert f.exists() == bool(want)
        if want:
            got = torch.frombuffer(bytearray(f.read_bytes()), dtype=torch.float32).view(len(want), -1)
            assert U.err(got, torch.stack(want)) < U.TOL[getattr(torch, dtype)], s["step"]


def test_generation_command(cuda, tmp_path, capsys):
    """The generation example on a model folder, in both types."""
    from tpp_pytorch_extension_b200.examples import run_generation
    cfg, w = U.model("odd", seed=8)
    U.save_folder(tmp_path, cfg, w)
    for dtype in ("float32", "bfloat16"):
        run_generation.main(["--model-dir", str(tmp_path), "--dtype", dtype, "--batch-size", "2", "--input-tokens", "20", "--max-new-tokens", "12",
                             "--num-iter", "1"])
        line = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
        assert line["model"] == "Vedizen" and line["weight_dtype"] == dtype and line["layers"] == len(cfg["layers"])

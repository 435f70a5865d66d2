"""The hybrid decoder's kernels, cache and runner against the plain implementation of oracle/hybrid_plain.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

from oracle import hybrid_plain as P
from tests import hybrid_util as U

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def portions(n, sizes):
    """n tokens cut into the given sizes, the last size repeating."""
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[min(i, len(sizes) - 1)], n - sum(out)))
        i += 1
    return out


CUTS = [[10 ** 6], [1], [2], [3, 1, 17], [64, 1], [33, 32, 5]]


# ---------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("M,N,K", [(1, 5, 3), (3, 130, 72), (16, 64, 200), (17, 33, 45), (70, 129, 64), (300, 70, 264)])
def test_linear_32_bit(cuda, M, N, K):
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    g = torch.Generator().manual_seed(M * N + K)
    x, w, b = (torch.randn(*s, generator=g, dtype=torch.float64).float() for s in ((M, K + 3), (N, K), (N,)))
    xd = x.to(cuda)[:, 2:2 + K]
    z = x[:, 2:2 + K].double() @ w.double().T + b.double()
    assert U.err(HL.linear(xd, w.to(cuda), b.to(cuda)), z) < 5e-6
    t = z.clone()
    t[:, N // 2:] = torch.tanh(t[:, N // 2:])
    assert U.err(HL.linear(xd, w.to(cuda), b.to(cuda), act="tanh", act_from=N // 2), t) < 5e-6
    a = torch.tensor([0.7, -0.4]).double()
    ap = torch.stack([P.softplus(a[0]), 0.5 + P.softplus(a[1])]).float().to(cuda)
    assert U.err(HL.linear(xd, w.to(cuda), b.to(cuda), act="xielu", act_params=ap), P.xielu(z, a)) < 5e-6


@pytest.mark.parametrize("M,N,K", [(1, 136, 8), (5, 200, 72), (40, 96, 264), (130, 264, 320), (1, 512, 4096), (33, 256, 2048)])
def test_linear_bf16_strided(cuda, M, N, K):
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    g = torch.Generator().manual_seed(M * N + K)
    x, w = torch.randn(M, K + 8, generator=g).to(torch.bfloat16), (torch.randn(N, K, generator=g) * K ** -0.5).to(torch.bfloat16)
    b = torch.randn(N, generator=g)
    xd = x.to(cuda)[:, 8:]
    z = x[:, 8:].double() @ w.double().T + b.double()
    assert U.err(HL.linear(xd, w.to(cuda), b.to(cuda), out_f32=True), z) < 1e-5
    assert U.err(HL.linear(xd, w.to(cuda), b.to(cuda)), z) < 5e-3
    a = torch.tensor([-0.3, 0.9]).double()
    ap = torch.stack([P.softplus(a[0]), 0.5 + P.softplus(a[1])]).float().to(cuda)
    assert U.err(HL.linear(xd, w.to(cuda), b.to(cuda), act="xielu", act_params=ap, out_f32=True), P.xielu(z, a)) < 1e-5


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 7])
@pytest.mark.parametrize("D", [20, 96, 517])
def test_postnorm_conv(cuda, taps, D):
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    g = torch.Generator().manual_seed(taps * D)
    B, S, eps, alpha = 3, 41, 1e-3, 1.3
    x, y = (torch.randn(B, S, D, generator=g) for _ in range(2))
    w, conv = torch.randn(D, generator=g) * 0.3, torch.randn(D, taps, generator=g)
    start = torch.tensor([0, 5, 18], dtype=torch.int32)
    want_x, want_h = torch.zeros(B, S, D).double(), torch.zeros(B, S, D).double()
    for b in range(B):
        n = int(start[b])
        v = P.zero_centred_norm(alpha * x[b, n:].double() + y[b, n:].double(), w.double(), eps)
        want_x[b, n:] = v
        want_h[b, n:] = v + P.causal_conv(v, conv.double())
    x[1, :5] = float("nan")  # padding holds anything
    norms = HL.Norms(eps, alpha, torch.float32)
    cw = conv.t().contiguous().to(cuda)
    for cut in CUTS:
        state = torch.zeros(B, taps - 1, D, device=cuda)
        xs, hs, t = [], [], 0
        for n in portions(S, cut):
            s = HL.Stream(B, n, x=x[:, t:t + n].reshape(-1, D).contiguous().to(cuda), y=y[:, t:t + n].reshape(-1, D).contiguous().to(cuda), w=w.to(cuda))
            xo, h = norms.enter(s, cw, state, start.to(cuda), None, t)
            assert h.shape[1] % 8 == 0 and not h[:, D:].any()
            xs.append(xo.view(B, n, D))
            hs.append(h[:, :D].reshape(B, n, D))
            t += n
        assert U.err(torch.cat(xs, 1), want_x) < 1e-5 and U.err(torch.cat(hs, 1), want_h) < 1e-5, cut


def mixer_over(mixers, h, cut, cuda, dtype):
    """Mixers 0 and (optionally) 1 that shares its latents, run over h [T, D] in portions; returns the last one's output."""
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    from tpp_pytorch_extension_b200._C._tpp_attn import TppCache
    cache, outs, t = TppCache(), [], 0
    start = torch.zeros(1, dtype=torch.int32, device=cuda)
    hd = torch.nn.functional.pad(h.float(), (0, -h.shape[1] % 8)).to(cuda, dtype)
    for n in portions(h.shape[0], cut):
        for i, m in enumerate(mixers):
            lc = cache.hybrid_layer(i)
            out = m.forward(hd[t:t + n].contiguous(), lc, cache, HL.Step(1, n, t, start, None))
            lc.offset += n
        outs.append(out)
        t += n
    return torch.cat(outs, 0)


def latent_mixer(cfg, w, i, cuda, dtype):
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    from tpp_pytorch_extension_b200.llm import fused_dofivik_infer as FD
    shape = FD.DofivikShape.from_config(cfg)
    lw = {k[3:]: v.float() for k, v in w.items() if k.startswith(f"l{i}.")}
    return FD.make_layer(shape, i, lw, HL.Norms(shape.norm_eps, shape.postln_alpha, dtype), cuda).mixer


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 31, 32, 33, 40, 64, 65, 1000])
def test_latent_attention_alone(cuda, dtype, window):
    """Own latents, then a layer that shares them with a longer and one with a shorter window; high gain so that single
    keys dominate and an edge that is one token off shows."""
    for other in (window + 3, max(1, window - 1)):
        cfg = U.config([U.attn(window=window, mlp=None), U.attn(window=other, kv_from=0, heads=2, vdim=9, mlp=None)])
        w = P.random_model(cfg, seed=window, gain=2.5)
        T = 150
        h = torch.randn(T, cfg["width"], generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).double()
        m0, m1 = cfg["layers"][0]["mixer"], cfg["layers"][1]["mixer"]
        lat = P.latent_of(w, "l0", m0, h, cfg["norm"]["eps"])
        want = [P.latent_attention(w, "l0", m0, h, lat, cfg["norm"]["eps"]), P.latent_attention(w, "l1", m1, h, lat, cfg["norm"]["eps"])]
        off = dict(m0, mask={"size": window + 1})
        assert window == 1000 or U.err(P.latent_attention(w, "l0", off, h, lat, cfg["norm"]["eps"]), want[0]) > 2 * U.TOL[dtype]
        mix = [latent_mixer(cfg, w, i, cuda, dtype) for i in range(2)]
        for cut in CUTS:
            assert U.err(mixer_over(mix[:1], h, cut, cuda, dtype), want[0]) < U.TOL[dtype], (cut, "own")
            assert U.err(mixer_over(mix, h, cut, cuda, dtype), want[1]) < U.TOL[dtype], (cut, "shared")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [dict(heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=96), dict(heads=1, dim=8, rot_dim=2, vdim=1, kv_rank=1, q_rank=1),
                                   dict(heads=16, dim=64, rot_dim=64, vdim=64, kv_rank=128, q_rank=64), dict(heads=3, dim=48, rot_dim=24, vdim=72, kv_rank=80, q_rank=50),
                                   dict(heads=17, dim=192, rot_dim=16, vdim=200, kv_rank=96, q_rank=40)])
def test_latent_attention_sizes(cuda, dtype, sizes):
    cfg = U.config([U.attn(window=70, scale=sizes["dim"] ** -0.5, mlp=None, **sizes)])
    w = P.random_model(cfg, seed=3, gain=1.5)
    h = torch.randn(200, cfg["width"], generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).double()
    m = cfg["layers"][0]["mixer"]
    want = P.latent_attention(w, "l0", m, h, P.latent_of(w, "l0", m, h, cfg["norm"]["eps"]), cfg["norm"]["eps"])
    mix = latent_mixer(cfg, w, 0, cuda, dtype)
    for cut in ([10 ** 6], [150, 1], [90, 60, 2]):
        assert U.err(mixer_over([mix], h, cut, cuda, dtype), want) < U.TOL[dtype], cut


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention_single_far_key(cuda, dtype):
    """One key per sequence stands out by far: positions inside its window return its value, the first one outside does not."""
    W, T, at = 45, 130, 37
    cfg = U.config([U.attn(heads=1, window=W, mlp=None)])
    w = P.random_model(cfg, seed=5)
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    g = torch.Generator().manual_seed(2)
    h0 = torch.randn(cfg["width"], generator=g).double()
    h = h0 + 0.05 * torch.randn(T, cfg["width"], generator=g).double()
    # all queries nearly equal; the token `at` gets the latent whose key points along that query
    q0 = (P.rms(h0 @ w["l0.mix.dq"].T, eps) * w["l0.mix.dq.norm"]) @ w["l0.mix.uq"].T
    h[at] = torch.linalg.pinv(w["l0.mix.dkv"][:m["kv_rank"]]) @ (w["l0.mix.uk"].T @ q0[:m["dim"]])
    w["l0.mix.uk"] *= 8.0
    h = h.to(torch.bfloat16).double()
    lat = P.latent_of(w, "l0", m, h, eps)
    want = P.latent_attention(w, "l0", m, h, lat, eps)
    for size, t in ((W - 1, at + W - 1), (W + 1, at + W)):  # the edge decides the output there
        assert U.err(P.latent_attention(w, "l0", dict(m, mask={"size": size}), h, lat, eps)[t:t + 1], want[t:t + 1]) > 0.3
    mix = latent_mixer(cfg, w, 0, cuda, dtype)
    for cut in ([10 ** 6], [at + 1, 1], [at + W, 1], [100, 2], [1]):
        got = mixer_over([mix], h, cut, cuda, dtype)
        for t in (at, at + 1, at + W - 1, at + W, T - 1):
            assert U.err(got[t:t + 1], want[t:t + 1]) < 2 * U.TOL[dtype], (cut, t)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim", [(2, 8), (3, 20), (1, 32), (2, 48), (4, 64), (2, 96), (2, 128), (1, 160), (1, 256)])
def test_general_delta_alone(cuda, dtype, heads, dim):
    cfg = U.config([U.delta(heads, dim, decay_rank=11)])
    w = P.random_model(cfg, seed=dim)
    T = 70 if dim <= 128 else 40
    h = torch.randn(T, cfg["width"], generator=torch.Generator().manual_seed(dim)).to(torch.bfloat16).double()
    want = P.general_delta(w, "l0", cfg["layers"][0]["mixer"], h, cfg["norm"]["eps"])
    mix = latent_mixer(cfg, w, 0, cuda, dtype)
    for cut in CUTS:
        assert U.err(mixer_over([mix], h, cut, cuda, dtype), want) < U.TOL[dtype], cut


@pytest.mark.parametrize("heads,dim", [(2, 64), (1, 128), (3, 40)])
def test_general_delta_long_memory(cuda, heads, dim):
    """Slow decay (close to one) and rates near zero or one over a long sequence: the state keeps what was written far back."""
    cfg = U.config([U.delta(heads, dim)])
    w = P.random_model(cfg, seed=1)
    w["l0.mix.w0"] -= 6.0
    w["l0.mix.a.b"] = torch.where(torch.arange(heads * dim) % 2 == 0, 4.0, -4.0).double()
    h = torch.randn(600, cfg["width"], generator=torch.Generator().manual_seed(3)).to(torch.bfloat16).double()
    want = P.general_delta(w, "l0", cfg["layers"][0]["mixer"], h, cfg["norm"]["eps"])
    for dtype in DTYPES:
        mix = latent_mixer(cfg, w, 0, cuda, dtype)
        for cut in ([10 ** 6], [500, 1], [37]):
            assert U.err(mixer_over([mix], h, cut, cuda, dtype), want) < U.TOL[dtype], (dtype, cut)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [1, 50, 72])
def test_dense_xielu(cuda, dtype, ff):
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    cfg = U.config([U.delta(mlp=ff)], width=45)
    w = P.random_model(cfg, seed=ff)
    h = (3 * torch.randn(33, 45, generator=torch.Generator().manual_seed(1))).to(torch.bfloat16).double()
    m = {k[3 + 4:]: v.float() for k, v in w.items() if k.startswith("l0.mlp.")}
    mlp = HL.DenseMlp({"up": m["up"], "up_bias": m["up.b"], "down": m["down"], "down_bias": m["down.b"], "act_params": m["act"]}, "xielu", dtype, cuda)
    hd = torch.nn.functional.pad(h.float(), (0, 3)).to(cuda, dtype)
    assert U.err(mlp.forward(hd), P.dense_mlp(w, "l0", h)) < U.TOL[dtype]


def test_argmax_f32(cuda):
    from tpp_pytorch_extension_b200._C import _hybrid_layers as HL
    x = torch.randn(7, 1001, device=cuda)
    x[2, 17] = x[2, 900] = 50.0
    x[3] = -5.0
    x[4, 33] = float("nan")
    assert torch.equal(HL.argmax_rows_f32(x), torch.argmax(x, dim=-1))
    assert HL.argmax_rows_f32(x[:, :3].contiguous()).shape == (7,)


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
        for t in range(40, 90):
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
    width = max(lens)

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


def test_long_decoding_passes_every_window(cuda):
    """Decoding far beyond every window, in the recorded step: the tokens of generate() equal those of fresh prefills."""
    cfg, w = U.model(U.config([U.attn(window=33), U.delta(2, 32), U.attn(window=64, kv_from=0), U.attn(window=5, mlp=None)]), seed=2, gain=2.0)
    r = U.runner_of(cfg, w, torch.float32)
    prompt, new = U.tokens(cfg, 6), 300
    out = r.generate(torch.tensor([prompt], device=cuda), new)[0].cpu().tolist()
    assert all(lc.pages() <= lc.window_pages() for lc in r._session.cache.get_cpp().layers if lc.arenas)
    lg = P.forward(cfg, w, out)
    for t in range(len(prompt) - 1, len(out) - 1):
        top = lg[t].topk(2)
        if float(top.values[0] - top.values[1]) > 1e-3:
            assert out[t + 1] == int(top.indices[0]), t


def test_beam_search_first_beam(cuda):
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


def test_bad_input_is_refused(cuda):
    cfg, w = U.model("one")
    r = U.runner_of(cfg, w, torch.float32)
    with pytest.raises(ValueError):
        r.forward(torch.tensor([[cfg["vocab"]]], device=cuda))
    _, cache = r.forward(torch.tensor([[1, 2]], device=cuda))
    with pytest.raises(ValueError):
        r.forward(torch.tensor([[1], [2]], device=cuda), None, None, cache)
    with pytest.raises(Exception):
        cache.crop(1)


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
        assert line["model"] == "Dofivik" and line["weight_dtype"] == dtype and line["layers"] == len(cfg["layers"])

"""CPU tests of the hybrid decoder: the plain implementation's own properties (every mechanism's edge shows in it), the
config and tensor-file readers, the registry and the host side of the page cache."""
import copy
import json

import pytest
import torch

from oracle import hybrid_plain as P
from tests import hybrid_util as U


def test_plain_window_edge_and_far_key():
    """A key that stands out is seen up to window - 1 tokens later and not one token further."""
    T, w = 30, 9
    q, k, v = torch.zeros(T, 1, 4).double(), torch.zeros(T, 1, 4).double(), torch.zeros(T, 1, 2).double()
    q[:, 0, 0] = 1.0
    k[5, 0, 0] = 50.0
    v[5, 0, 0] = 1.0
    o = P.window_attention(q, k, v, 1.0, w)[:, 0, 0]
    assert torch.all(o[5:5 + w] > 0.99) and torch.all(o[5 + w:] == 0) and torch.all(o[:5] == 0)


def test_plain_rotation_is_relative():
    g = torch.Generator().manual_seed(0)
    q, k = torch.randn(1, 8, generator=g).double(), torch.randn(1, 8, generator=g).double()
    at = lambda x, p: P.rotate_pairs(x, torch.tensor([p]), 300.0)
    assert torch.allclose((at(q, 20) * at(k, 13)).sum(), (at(q, 7) * at(k, 0)).sum())
    assert not torch.allclose((at(q, 20) * at(k, 13)).sum(), (at(q, 8) * at(k, 0)).sum())


def test_plain_conv_and_delta_small_cases():
    h = torch.tensor([[1.0], [10.0], [100.0]]).double()
    w = torch.tensor([[3.0, 2.0]]).double()
    assert P.causal_conv(h, w).flatten().tolist() == [2.0, 23.0, 230.0]
    S = torch.eye(2).double() * 2
    k, v, r = (torch.tensor(x).double() for x in ([3.0, 4.0], [1.0, 0.0], [0.0, 1.0]))
    S2, o = P.delta_step(S, r, k, v, torch.full((2,), 0.5).double(), torch.ones(2).double())
    u = k / torch.sqrt(torch.tensor(25.000001).double())
    want = 0.5 * S - torch.outer(u, u @ S) + torch.outer(k, v)
    assert torch.allclose(S2, want) and torch.allclose(o, want[1])


def test_plain_model_mistakes_show():
    """A window that is one token off, a missing gate, a dropped shared latent or state changes the logits visibly."""
    cfg, w = U.model("mixed", gain=3.0)
    t = U.tokens(cfg, 50)
    base = P.forward(cfg, w, t)

    def change(mut):
        c, ww = copy.deepcopy(cfg), dict(w)
        mut(c, ww)
        return U.err(P.forward(c, ww, t), base)

    assert change(lambda c, ww: c["layers"][0]["mixer"]["mask"].update(size=38)) > 1e-3
    assert change(lambda c, ww: c["layers"][4]["mixer"]["mask"].update(size=32)) > 1e-3
    assert change(lambda c, ww: c["layers"][2]["mixer"]["rot"].update(base=5001.0)) > 1e-5
    assert change(lambda c, ww: ww.update({"l0.mix.g": w["l0.mix.g"] * 0})) > 1e-2
    assert change(lambda c, ww: ww.update({"l3.canon2": w["l3.canon2"] * 0})) > 1e-2
    assert change(lambda c, ww: ww.update({"l1.mix.w0": w["l1.mix.w0"] + 1.0})) > 1e-3


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_tensor_names_of_a_config(name):
    from tpp_pytorch_extension_b200.llm import fused_dofivik_infer as FD
    cfg, w = U.model(name)
    ranks = {l["mixer"].get("decay_rank", 8) for l in cfg["layers"] if l["type"] == "general_delta"}
    shapes = FD.tensor_shapes(FD.DofivikShape.from_config(cfg), 8)
    assert set(shapes) == set(w)
    for n, s in shapes.items():
        if ranks == {8} or not n.endswith((".w1", ".w2")):
            assert tuple(w[n].shape) == s, n


def test_config_reader_refuses_what_it_does_not_know():
    from tpp_pytorch_extension_b200.llm.fused_dofivik_infer import DofivikShape
    for mut in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="experts"),
                lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4), lambda c: c["layers"][2]["mixer"].update(kv_from=1),
                lambda c: c["layers"][2]["mixer"].update(kv_from=3), lambda c: c["layers"][2]["mixer"].update(kv_rank=16)):
        c = copy.deepcopy(U.CONFIGS["mixed"])
        mut(c)
        with pytest.raises(ValueError):
            DofivikShape.from_config(c)
    s = DofivikShape.from_config(U.CONFIGS["mixed"])
    assert [s.cache_window(i) for i in (0, 2, 4)] == [70, 70, 33]


def test_safetensors_round_trip(tmp_path):
    from tpp_pytorch_extension_b200.utils import safetensors_file as S
    t = {"b": torch.arange(5, dtype=torch.int8), "a": torch.randn(3, 4).to(torch.bfloat16), "i": torch.arange(7, dtype=torch.int32),
         "e": torch.empty(0, 4), "f": torch.randn(2, 2)}
    S.save(tmp_path / "x.safetensors", t)
    got = S.load(tmp_path / "x.safetensors")
    assert list(got) == list(t) and all(got[k].dtype == t[k].dtype and torch.equal(got[k], t[k]) for k in t)


def test_registry(tmp_path):
    from tpp_pytorch_extension_b200.llm import model_registry as R
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Dofivik"}))
    assert R.architecture_of(tmp_path) == "Dofivik" and torch.float32 in R.dtypes_of("Dofivik")
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["LlamaForCausalLM"]}))
    assert R.architecture_of(tmp_path) == "LlamaForCausalLM" and torch.float32 not in R.dtypes_of("LlamaForCausalLM")
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    with pytest.raises(ValueError):
        R.architecture_of(tmp_path)


@pytest.mark.parametrize("window", [1, 2, 31, 32, 33, 34, 64, 65, 100])
def test_window_pages_suffice_and_are_few(window):
    from tpp_pytorch_extension_b200._C._tpp_attn import HybridLayerCache
    lc = HybridLayerCache()
    lc.window = window
    n = lc.window_pages()
    touched = max(t // 32 - max(t - window + 1, 0) // 32 + 1 for t in range(400))
    assert touched == n
    for t in range(200):  # tokens of one window never share a (page, row)
        seen = {(j // 32 % n, j % 32) for j in range(max(t - window + 1, 0), t + 1)}
        assert len(seen) == min(window, t + 1)


def test_page_table_growth_and_states():
    from tpp_pytorch_extension_b200._C._tpp_attn import HybridLayerCache, TppCache
    c = TppCache()
    lc = c.hybrid_layer(0)
    lc.ensure_latent(2, 16, 10, 200, torch.float32, "cpu")
    first = lc.arenas[0].data_ptr()
    assert lc.pages() >= 1 and lc.capacity() < 200
    while lc.offset < 600:
        lc.ensure_latent(2, 16, 50, 200, torch.float32, "cpu")
        lc.offset += 50
    assert lc.pages() == lc.window_pages() and lc.arenas[0].data_ptr() == first and lc.fits(2, 10 ** 6)
    s = lc.state("x", (2, 3), "cpu")
    s.copy_(torch.arange(6).view(2, 3))
    lc.arenas[0][:, 1] = 7.0
    c.start = torch.tensor([0, 4], dtype=torch.int32)
    c.keep_sequences([1])
    assert lc.states["x"].tolist() == [[3.0, 4.0, 5.0]] and c.start.tolist() == [4] and float(lc.arenas[0].min()) == 7.0
    assert lc.batch() == 1 and lc.ptrs[0].item() == lc.arenas[0].data_ptr()
    c.reorder_cache(torch.tensor([0, 0, 0]))
    assert lc.states["x"].shape == (3, 3) and c.start.tolist() == [4, 4, 4]
    with pytest.raises(Exception):
        c.crop(5)
    c.reset()
    assert lc.offset == 0 and not lc.states["x"].any() and c.start is None


def test_left_padding_only():
    from tpp_pytorch_extension_b200.llm.fused_dofivik_infer import DofivikRunner
    assert DofivikRunner._padding(torch.tensor([[0, 0, 1], [1, 1, 1]])).tolist() == [2, 0]
    with pytest.raises(ValueError):
        DofivikRunner._padding(torch.tensor([[1, 0, 1]]))


def test_trace_batches(tmp_path):
    """Rows, masks and wanted places of a replayed trace (a stand-in runner that returns the token ids as logits)."""
    from tpp_pytorch_extension_b200.examples.trace_run import TraceBatch

    class Cpp:
        def keep_sequences(self, rows):
            self.kept = rows

    class Cache:
        cpp = Cpp()

        def get_cpp(self):
            return self.cpp

    class Runner:
        embed = torch.zeros(1)

        def forward(self, ids, mask, pos, cache):
            self.seen = (ids, mask, pos)
            return ids.reshape(-1)[self.logit_rows].unsqueeze(-1), Cache()

    b = TraceBatch(Runner())
    got = b.step([{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}, {"id": "b", "tokens": [9], "want": [0]}])
    assert got.flatten().tolist() == [5, 7, 9]
    assert b.runner.seen[1].tolist() == [[1, 1, 1], [0, 0, 1]] and b.runner.seen[2].tolist() == [[0, 1, 2], [0, 0, 0]]
    got = b.step([{"id": "b", "tokens": [4], "want": [0]}, {"id": "a", "tokens": [3], "want": []}])
    assert got.flatten().tolist() == [4] and b.runner.seen[0].tolist() == [[3], [4]] and b.runner.seen[2].tolist() == [[3], [1]]
    b.end(["a"])
    assert b.rows == ["b"] and b.cache.get_cpp().kept == [1]
    with pytest.raises(ValueError):
        b.step([{"id": "c", "tokens": [1], "want": []}])
    b.end(["b"])
    assert not b.rows and b.step([{"id": "c", "tokens": [1], "want": [0]}]).tolist() == [[1]]

"""CPU tests of the Vedizen decoder: the plain implementation's own properties (every mechanism's edge shows in it), the
config reader, the order of layer runs, the registry, and the host side of its cache."""
import copy
import json
import math

import pytest
import torch

from oracle import vedizen_plain as P
from tests import vedizen_util as U


def test_plain_recurrence_small_case():
    q, k, v, a = (torch.tensor(x).double() for x in ([[1.0, 2.0], [3.0, 1.0]], [[1.0, 0.0], [2.0, 1.0]], [[5.0], [7.0]], [[0.9, 0.9], [0.5, 0.25]]))
    # S1 = [5, 0]; S2 = [2.5 + 14, 0 + 7]
    assert torch.allclose(P.gla_recurrence(q, k, v, a), torch.tensor([[5.0], [3 * 16.5 + 7]]).double())


def test_plain_chunk_edge_and_far_key():
    """A key that stands out is seen up to the end of its chunk and not by the next chunk's first token."""
    T, C, at = 30, 9, 11
    q, k, v = torch.zeros(T, 4).double(), torch.zeros(T, 4).double(), torch.zeros(T, 2).double()
    q[:, 0], k[at, 0], v[at, 0] = 1.0, 50.0, 1.0
    o = P.attention_map(q, k, v, 1.0, 100.0, C)[:, 0]
    assert torch.all(o[at:18] > 0.99) and torch.all(o[18:] == 0) and torch.all(o[:at] == 0)


def test_plain_cap_bounds_the_scores():
    q, k, v = torch.ones(2, 1).double(), torch.tensor([[0.0], [1e4]]).double(), torch.tensor([[0.0], [1.0]]).double()
    p = P.attention_map(q, k, v, 1.0, 2.0, 10)[1, 0]
    assert abs(float(p / (1 - p)) - 2.718281828 ** 2) < 1e-6


def test_plain_clamps():
    w = {"m.gate": torch.eye(1).double(), "m.up": -3 * torch.eye(1).double(), "m.down": torch.eye(1).double()}
    at = lambda x: float(P.clamped_glu(torch.tensor([[x]]).double(), w, "m", 2.0))
    s = lambda g: g / (1.0 + math.exp(-1.702 * g))
    assert abs(at(5.0) - s(2.0) * -1.0) < 1e-12 and abs(at(-5.0) - s(-5.0) * 3.0) < 1e-12 and abs(at(0.5) - s(0.5) * -0.5) < 1e-12


def test_plain_model_mistakes_show():
    """A chunk that is one token off, a dropped step vector, pass, bias, map or decay changes the logits visibly."""
    cfg, w = U.model("mixed", gain=3.0)
    t = U.tokens(cfg, 80)
    base = P.forward(cfg, w, t)

    def change(mut):
        c, ww = copy.deepcopy(cfg), dict(w)
        mut(c, ww)
        return U.err(P.forward(c, ww, t), base)

    assert change(lambda c, ww: c["layers"][1]["mixer"]["mask"].update(size=38)) > 1e-2
    assert change(lambda c, ww: c["layers"][3]["mixer"]["mask"].update(size=63)) > 1e-2
    assert change(lambda c, ww: c["layers"][1]["mixer"].update(softcap=9.5)) > 1e-3
    assert change(lambda c, ww: c["layers"][1]["mixer"].update(diff=0.31)) > 1e-3
    assert change(lambda c, ww: c["loop"].update(times=2)) > 1e-2
    assert change(lambda c, ww: ww.update({"loop.step": w["loop.step"].roll(1, 0)})) > 1e-2
    assert change(lambda c, ww: ww.update({"l1.mix.k.b": w["l1.mix.k.b"] * 0})) > 1e-3
    assert change(lambda c, ww: ww.update({"l1.mix.lq2": w["l1.mix.lq2"] * 0})) > 1e-4
    assert change(lambda c, ww: ww.update({"l0.mix.a2.b": w["l0.mix.a2.b"] + 0.5})) > 1e-3
    assert change(lambda c, ww: c["layers"][0]["mlp"].update(limit=1.0)) > 1e-4
    assert change(lambda c, ww: ww.update({"l2.norm1.b": w["l2.norm1.b"] * 0})) > 1e-2


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_tensor_names_of_a_config(name):
    from tpp_pytorch_extension_b200.llm import fused_vedizen_infer as FV
    cfg, w = U.model(name)
    shapes = FV.tensor_shapes(FV.VedizenShape.from_config(cfg), 5)
    assert set(shapes) == set(w)
    assert all(tuple(w[n].shape) == s for n, s in shapes.items())


@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 3, 2), (1, 2, 3), (2, 3, 2)])
def test_order_of_runs(loop):
    from tpp_pytorch_extension_b200.llm.fused_vedizen_infer import VedizenShape
    cfg = U.config([U.gla(), U.attn(), U.gla()], loop=loop)
    assert VedizenShape.from_config(cfg).runs() == P.layer_runs(cfg)
    if loop == (1, 2, 3):
        assert P.layer_runs(cfg) == [(0, None), (1, 0), (1, 1), (1, 2), (2, None)]


def test_config_reader_refuses_what_it_does_not_know():
    from tpp_pytorch_extension_b200.llm.fused_vedizen_infer import VedizenShape
    for mut in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="experts"),
                lambda c: c["loop"].update(stop=9), lambda c: c["loop"].update(start=4), lambda c: c["loop"].update(times=0)):
        c = copy.deepcopy(U.CONFIGS["mixed"])
        mut(c)
        with pytest.raises(ValueError):
            VedizenShape.from_config(c)


def test_registry_and_components(tmp_path):
    from tpp_pytorch_extension_b200 import _build
    from tpp_pytorch_extension_b200.llm import model_registry as R
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Vedizen"}))
    assert R.architecture_of(tmp_path) == "Vedizen" and R.dtypes_of("Vedizen") == (torch.bfloat16, torch.float32)
    assert not R.quantizes("Vedizen") and not R.quantizes("Dofivik") and R.quantizes("LlamaForCausalLM")
    names = {s.rsplit("tpx_", 1)[1][:-3] for s in _build.sources()}
    assert all(set(c) <= names for c in _build.COMPONENTS.values())


def test_pages_of_keys_and_values():
    """Pages with a head dimension: growth moves nothing, a chunk's table stops growing, sequences end and are repeated."""
    from tpp_pytorch_extension_b200._C._tpp_attn import TppCache
    c = TppCache()
    lc = c.hybrid_layer(0)
    slab = (2, 3, 32, 24)
    lc.ensure_pages(slab, 10, 150, torch.float32, "cpu")
    first = lc.arenas[0].data_ptr()
    while lc.offset < 500:
        lc.ensure_pages(slab, 40, 150, torch.float32, "cpu")
        lc.offset += 40
    assert lc.pages() == lc.window_pages() == 6 and lc.arenas[0].data_ptr() == first and lc.batch() == 2
    assert lc.ptrs.tolist()[:2] == [first, first + 2 * 3 * 32 * 24 * 4]
    with pytest.raises(Exception):
        lc.ensure_pages((2, 3, 32, 40), 1, 150, torch.float32, "cpu")
    lc.reserve(10000)
    assert lc.pages() == 6 and lc.fits(2, 10 ** 6)
    for a in lc.arenas:
        a[:, 1] = 7.0
    c.start = torch.tensor([0, 4], dtype=torch.int32)
    c.keep_sequences([1])
    assert lc.batch() == 1 and all(float(a.min()) == 7.0 for a in lc.arenas) and lc.ptrs[0].item() == lc.arenas[0].data_ptr()
    # a chunk never meets one of its own rows again
    n = lc.window_pages()
    for t in range(700):
        seen = [(j // 32 % n, j % 32) for j in range(t // 150 * 150, t + 1)]
        assert len(set(seen)) == len(seen)

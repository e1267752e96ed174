"""The Fopezen decoder without a GPU: configuration (round trip, absent keys, errors that name the key), the layout's parts and
tensor names, which pages a window that keeps the first positions gives back, the tables of the position vector, and the
plain statement against values worked by hand."""
import copy
import json
import math

import pytest
import torch

import plain_fopezen as plain
from scriptling_llm_lib_b200 import models  # noqa: F401
from scriptling_llm_lib_b200.cache.needs import PAGE, CacheNeed
from scriptling_llm_lib_b200.cache.store import SequenceCache
from scriptling_llm_lib_b200.config.base import ConfigError
from scriptling_llm_lib_b200.config.fopezen import FopezenConfig
from scriptling_llm_lib_b200.config.registry import architecture_for
from scriptling_llm_lib_b200.engine.model import DecoderModel

RAW = {
    "architecture": "Fopezen", "vocab": 70, "width": 40, "norm": {"eps": 1e-5},
    "layers": [
        {"type": "attention", "mixer": {"dim": 6, "heads": 3, "kv_heads": 1, "scale": 0.3, "v_mix": False, "vdim": 5},
         "mlp": {"ff": 20, "kind": "dense"}},
        {"type": "attention_2", "mixer": {"dim": 8, "heads": 4, "kv_heads": 2, "mask": {"keep_first": 3, "size": 17}, "scale": 0.2,
                                          "v_mix": True, "vdim": 6}, "mlp": None},
        {"type": "attention", "mixer": {"dim": 10, "heads": 6, "kv_heads": 3, "mask": {"keep_first": 0, "size": 90}, "scale": 0.5,
                                        "v_mix": True, "vdim": 4}, "mlp": {"ff": 12, "kind": "dense"}},
    ],
}


def test_the_configuration_reads_back_as_it_was_written():
    cfg = FopezenConfig.from_dict(RAW, "t")
    assert cfg.to_json_dict() == RAW
    assert cfg.first_mixed == 1 and cfg.layers[0].mixer.window is None and cfg.layers[1].mlp is None
    assert FopezenConfig.from_dict(json.loads(json.dumps(cfg.to_json_dict())), "t") == cfg
    bare = copy.deepcopy(RAW)
    for l in bare["layers"]:
        l["mixer"].pop("v_mix")
        l["mixer"].pop("mask", None)
    c2 = FopezenConfig.from_dict(bare, "t")
    assert c2.first_mixed is None and all(l.mixer.window is None and l.mixer.keep_first == 0 for l in c2.layers)


@pytest.mark.parametrize("path,value,word", [
    (("layers", 1, "mixer", "kv_heads"), 3, "heads"), (("layers", 1, "mixer", "vdim"), 7, "v_mix"),
    (("layers", 1, "mixer", "mask", "size"), 0, "size"), (("layers", 1, "mixer", "mask", "keep_first"), -1, "keep_first"),
    (("layers", 0, "type"), "attention_3", "type"), (("norm", "eps"), 0, "eps"), (("layers", 0, "mlp", "kind"), "moe", "kind"),
    (("layers", 2, "mixer", "v_mix"), 1, "v_mix"), (("width",), 0, "width"), (("layers",), [], "layers"),
    (("layers", 0, "mixer", "scale"), None, "scale"), (("layers", 0, "mixer", "dim"), 513, "513"),
])
def test_errors_name_the_key(path, value, word):
    raw = copy.deepcopy(RAW)
    at = raw
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        FopezenConfig.from_dict(raw, "t")
    assert word in str(e.value)


def test_the_layout_names_the_designs_tensors_and_needs():
    arch = architecture_for("Fopezen")
    layout = arch.layout(arch.config_class.from_dict(RAW, "t"))
    model = DecoderModel(layout)
    shapes = {s.name: tuple(s.shape) for s in model.tensor_specs()}
    assert shapes["embed"] == (70, 40) and shapes["final.norm"] == (40,) and "head" not in shapes
    assert shapes["l0.mix.q"] == (18, 40) and shapes["l0.mix.q.b"] == (18,) and shapes["l0.mix.q.norm"] == (6,)
    assert shapes["l0.mix.k.norm"] == (6,) and shapes["l0.mix.v"] == (5, 40) and shapes["l0.mix.g"] == (15, 40)
    assert shapes["l0.mix.o"] == (40, 15) and shapes["l0.mix.o.b"] == (40,) and "l0.mix.vmix" not in shapes
    assert shapes["l1.mix.q.norm"] == (32,) and shapes["l1.mix.k.norm"] == (16,) and shapes["l1.mix.vmix"] == ()
    assert not {"l1.mix.g", "l1.mix.o.b", "l1.norm2", "l1.mlp.up"} & set(shapes) and shapes["l1.norm1"] == (40,)
    assert shapes["l2.mlp.up"] == (12, 40) and shapes["l2.mlp.down"] == (40, 12) and shapes["l2.mix.v.b"] == (12,)
    assert layout.ignorable_tensors == ("l0.mix.vmix",) and model.graph_safe()
    needs = model.cache_needs()
    assert needs[0].kind == "full" and needs[0].keep == 0 and needs[0].value_dim == 5
    assert (needs[1].kind, needs[1].window, needs[1].keep, needs[1].head_dim, needs[1].value_dim) == ("window", 17, 3, 8, 6)
    assert needs[2].keep == 0 and all(v is None for v in model.state_needs().values())


def test_a_window_gives_back_the_pages_between_the_kept_positions_and_itself():
    for window, keep, kept_pages in ((100, 0, 0), (100, 1, 1), (100, PAGE, 1), (100, PAGE + 1, 2), (30, 5, 1)):
        need = CacheNeed("window", 1, 4, window, keep=keep)
        cache = SequenceCache({0: need}, {}, 2, 12, torch.float32, "cpu")
        slot = cache.open()
        for length in range(1, 700):
            cache.reserve([(slot, 1)])
            cache.advance([(slot, 1)])
            pages = cache.groups[0].pages[slot]
            for j in range(length):                   # whatever the next query can see has its page
                if length - j < window or j < keep:
                    assert pages[j // PAGE] >= 0
            held = sum(p >= 0 for p in pages)
            assert held <= kept_pages + need.pages_seen() and cache.groups[0].pool.n_held == held
            seen = {j // PAGE for j in range(length + 1) if length - j < window or j < keep}
            assert len(seen) <= need.pages_seen()
        assert held <= kept_pages + (window + PAGE - 2) // PAGE + 1
        cache.close(slot)
        assert cache.groups[0].pool.n_held == 0
    with pytest.raises(ValueError):
        CacheNeed("window", 1, 4, 10, keep=-1)


def test_the_tables_of_the_position_vector():
    from scriptling_llm_lib_b200.parts.embedding import SinusoidEmbedding
    for width in (7, 16, 50):
        e = SinusoidEmbedding(10, width, "e")
        e.prepare(20000, "cpu")
        for p in (0, 1, 63, 64, 65, 4095, 12345, 19999):
            a, b = e.coarse[p // 64].double(), e.fine[p % 64].double()
            s, c = a[:, 0] * b[:, 1] + a[:, 1] * b[:, 0], a[:, 1] * b[:, 1] - a[:, 0] * b[:, 0]
            got = torch.stack([s, c], dim=-1).reshape(-1)[:width]
            assert float((got - plain.sinusoid(p, width)).abs().max()) < 3e-7


def test_parts_refuse_what_does_not_go_together():
    from scriptling_llm_lib_b200.parts.attention import Attention
    base = dict(hidden=8, n_heads=2, n_kv_heads=1, head_dim=4, position=None, q_name="q", k_name="k", v_name="v", o_name="o")
    for extra in (dict(keep_first=2), dict(sink_name="s", sink_value=0.0), dict(biases=dict(q_name="b")),
                  dict(qk_norm=dict(q_name="a", k_name="b", eps=1e-6, per="row")), dict(value_norm_eps=1e-6, keep_first=1, window=4),
                  dict(conv=dict(taps=2, q_name="a", k_name="b", v_name="c"), value_mix=dict(share_name="m", first=True))):
        with pytest.raises(ValueError):
            Attention(**base, **extra)
    assert not Attention(**base).general and Attention(**base, window=4, keep_first=1).general


def test_the_plain_statement_by_hand():
    s = plain.sinusoid(3, 4)
    assert torch.allclose(s, torch.tensor([math.sin(3), math.cos(3), math.sin(0.03), math.cos(0.03)], dtype=torch.float64))
    assert [j for j in range(12) if plain.sees(10, j, 4, 2)] == [0, 1, 7, 8, 9, 10]
    assert [j for j in range(12) if plain.sees(3, j, 4, 2)] == [0, 1, 2, 3] and plain.sees(900, 5, None, 0)
    w = plain.weights_of(torch.tensor([0.0, math.log(2.0)], dtype=torch.float64), True)
    assert torch.allclose(w, torch.tensor([0.25, 0.5], dtype=torch.float64))
    w = plain.weights_of(torch.tensor([0.0, math.log(3.0)], dtype=torch.float64), False)
    assert torch.allclose(w, torch.tensor([0.25, 0.75], dtype=torch.float64))
    x = torch.tensor([[3.0, 4.0, 0.0, 0.0]], dtype=torch.float64)
    ones = torch.ones(4, dtype=torch.float64)
    assert torch.allclose(plain.head_norms(x, ones, 2, 0.0, True), x / 2.5)
    per_head = plain.head_norms(x, ones[:2], 2, 1e-9, False)
    assert torch.allclose(per_head, torch.tensor([[3.0, 4.0, 0.0, 0.0]], dtype=torch.float64) / math.sqrt(12.5))
    assert torch.allclose(plain.shifted_rms_norm(x, torch.full((4,), -0.5, dtype=torch.float64), 0.0), x / 5.0)
    assert float(plain.mixed_values(torch.tensor(2.0), torch.tensor(10.0), torch.tensor(0.25))) == 4.0
    f = plain.feed_forward(torch.tensor([[1.0, -2.0]], dtype=torch.float64),
                           {"up": torch.tensor([[3.0, 0.0], [0.0, 1.0]], dtype=torch.float64), "down": torch.eye(2, dtype=torch.float64)}, "")
    assert torch.equal(f, torch.tensor([[9.0, 0.0]], dtype=torch.float64))

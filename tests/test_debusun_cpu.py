"""The Debusun decoder without a GPU: configuration (round trip, errors that name the key), the layout's parts, tensor names
and schedule, cache and state needs, and the plain statement against values worked by hand."""
import copy
import json
import math

import pytest
import torch

import plain_debusun as plain
from scriptling_llm_lib_b200 import models  # noqa: F401
from scriptling_llm_lib_b200.config.base import ConfigError
from scriptling_llm_lib_b200.config.debusun import DebusunConfig
from scriptling_llm_lib_b200.config.registry import architecture_for
from scriptling_llm_lib_b200.engine.model import DecoderModel
from scriptling_llm_lib_b200.parts.attention import Attention

F64 = torch.float64
RAW = {
    "architecture": "Debusun", "vocab": 70, "width": 40, "norm": {"eps": 1e-5},
    "embedding": {"bigram": {"buckets": 29, "mul_cur": 3, "mul_prev": 11}, "scale": 2.5}, "loop": {"start": 0, "stop": 2, "times": 3},
    "layers": [
        {"type": "mamba2", "mixer": {"conv": 3, "groups": 2, "heads": 6, "norm_groups": 3, "state": 9, "vdim": 5}, "mlp": None},
        {"type": "latent_attention", "mixer": {"dim": 6, "heads": 3, "kv_rank": 10, "mask": {"size": 33}, "rot_dim": 4, "scale": 0.3,
                                               "vdim": 5, "rot": {"base": 100.0, "dims": 4, "scaling": {
                                                   "factor": 3.0, "fast": 4.0, "original": 40, "slow": 1.0}}},
         "mlp": {"ff": 12, "kind": "dense"}},
        {"type": "attention", "mixer": {"dim": 8, "heads": 4, "kv_heads": 2, "mask": {"size": 21}, "scale": 0.5, "vdim": 4,
                                        "rot": {"base": 50.0, "dims": 6}},
         "mlp": {"ff": 20, "kind": "dense"}},
    ],
}


def test_the_configuration_reads_back_as_it_was_written():
    cfg = DebusunConfig.from_dict(RAW, "t")
    assert cfg.to_json_dict() == RAW
    assert DebusunConfig.from_dict(json.loads(json.dumps(cfg.to_json_dict())), "t") == cfg
    bare = {k: v for k, v in RAW.items() if k not in ("embedding", "loop")}
    c2 = DebusunConfig.from_dict(bare, "t")
    assert c2.bigram is None and c2.loop is None and c2.embedding_scale == 1.0 and cfg.layers[0].ff is None


@pytest.mark.parametrize("path,value,word", [
    (("layers", 2, "mixer", "kv_heads"), 3, "heads"), (("layers", 2, "mixer", "rot", "dims"), 5, "dims"),
    (("layers", 1, "mixer", "rot", "dims"), 6, "dims"), (("layers", 0, "mixer", "groups"), 4, "groups"),
    (("layers", 0, "mixer", "norm_groups"), 7, "norm_groups"), (("layers", 2, "mixer", "mask", "size"), 0, "size"),
    (("loop", "stop"), 4, "loop"), (("layers", 1, "type"), "scan", "type"), (("norm", "eps"), 0, "eps"),
    (("embedding", "bigram", "buckets"), 0, "buckets"), (("layers", 1, "mlp", "kind"), "moe", "kind"),
])
def test_errors_name_the_key(path, value, word):
    raw = copy.deepcopy(RAW)
    at = raw
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        DebusunConfig.from_dict(raw, "t")
    assert word in str(e.value)


def test_the_layout_names_the_designs_tensors_and_schedule():
    arch = architecture_for("Debusun")
    layout = arch.layout(arch.config_class.from_dict(RAW, "t"))
    model = DecoderModel(layout)
    shapes = {s.name: tuple(s.shape) for s in model.tensor_specs()}
    assert shapes["embed"] == (70, 40) and shapes["bigram"] == (30, 40) and shapes["loop.step"] == (3, 40) and shapes["head"] == (70, 40)
    assert shapes["l0.mix.in"] == (30 + 30 + 2 * 18 + 6, 40) and shapes["l0.mix.conv"] == (66, 3) and shapes["l0.mix.conv.b"] == (66,)
    assert shapes["l0.mix.dt_bias"] == shapes["l0.mix.A_log"] == shapes["l0.mix.D"] == (6,) and shapes["l0.mix.norm"] == (30,)
    assert shapes["l0.mix.o"] == (40, 30) and "l0.norm2" not in shapes and "l0.mlp.up" not in shapes
    assert shapes["l1.mix.q"] == (30, 40) and shapes["l1.mix.dkv"] == (14, 40) and shapes["l1.mix.dkv.norm"] == (10,)
    assert shapes["l1.mix.uk"] == (18, 10) and shapes["l1.mix.uv"] == (15, 10) and shapes["l1.mix.sink"] == (3,)
    assert shapes["l1.mix.g"] == (15, 40) and shapes["l1.mix.o"] == (40, 15) and shapes["l1.mlp.up"] == (12, 40)
    assert shapes["l2.mix.q"] == (32, 40) and shapes["l2.mix.k"] == (16, 40) and shapes["l2.mix.v"] == (8, 40)
    assert shapes["l2.mix.o"] == (40, 16) and "l2.mix.q.norm" not in shapes and shapes["final.norm"] == (40,)
    # the run of two layers three times; its vector before every pass, the embedding's output (part 3) before all but the first
    assert [(e.layer, e.cache_unit, e.before) for e in layout.schedule] == [
        (0, 0, (0,)), (1, 1, ()), (0, 2, (3, 1)), (1, 3, ()), (0, 4, (3, 2)), (1, 5, ()), (2, 6, ())]
    needs = model.cache_needs()
    assert needs[0] is None and needs[1] == needs[3] == needs[5]
    assert (needs[1].kind, needs[1].window, needs[1].head_dim, needs[1].value_dim) == ("window", 33, 14, 0)
    assert (needs[6].kind, needs[6].window, needs[6].kv_heads, needs[6].head_dim, needs[6].value_dim) == ("window", 21, 2, 8, 4)
    state = model.state_needs()
    assert state["embedding"].dtype == torch.int32 and state[2]["S"].shape == (6, 9, 5) and state[2]["conv"].shape == (2, 66)
    assert state[2]["S"].dtype == torch.float32 and model.graph_safe()
    once = copy.deepcopy(RAW)
    once["loop"]["times"] = 1
    one = arch.layout(arch.config_class.from_dict(once, "t"))
    assert [e.before for e in one.schedule] == [(0,), (), ()] and "keep_output" not in dict(one.embedding.params) or not one.embedding.params["keep_output"]


def test_a_norm_behind_the_rotation_has_no_weight_and_is_per_head():
    base = dict(hidden=16, n_heads=2, n_kv_heads=1, head_dim=8, position=None, q_name="q", k_name="k", v_name="v", o_name="o")
    with pytest.raises(ValueError):
        Attention(**base, qk_norm=dict(eps=1e-6, per="projection", after_rotation=True))
    with pytest.raises(ValueError):
        Attention(**base, qk_norm=dict(eps=1e-6, per="head"))
    with pytest.raises(ValueError):
        Attention(**base, qk_norm=dict(eps=1e-6, per="head", after_rotation=True, q_name="a", k_name="b"))
    assert Attention(**base, qk_norm=dict(eps=1e-6, per="head", after_rotation=True)).general


def test_the_plain_statement_by_hand():
    assert plain.pair_rows([5, 2, 9], 7, 3, 4) == [7, (5 * 3 + 2 * 4) % 7, (2 * 3 + 9 * 4) % 7]
    t = torch.tensor([[1.0, 2.0], [3.0, -1.0]], dtype=F64)
    p = torch.tensor([[10.0, 0.0], [0.0, 10.0], [5.0, 5.0]], dtype=F64)
    x = plain.embed([1, 0], t, 2.0, p, {"buckets": 2, "mul_prev": 1, "mul_cur": 0})
    assert x.tolist() == [[11.0, 3.0], [2.0, 14.0]]
    # the window holds the position itself and the size - 1 before it
    assert [plain.visible(i, 3) for i in range(5)] == [0, 0, 0, 1, 2] and plain.visible(9, None) == 0 and plain.visible(9, 1) == 9
    # neighbours turn; the angle of pair i is position * base^(-2i/dims)
    v = torch.zeros(2, 1, 5, dtype=F64)
    v[1, 0] = torch.tensor([1.0, 0.0, 0.0, 1.0, 7.0])
    r = plain.rotate(v, 4, 100.0)[1, 0]
    want = [math.cos(1), math.sin(1), -math.sin(0.1), math.cos(0.1), 7.0]
    assert torch.allclose(r, torch.tensor(want, dtype=F64))
    f, amp = plain.frequencies(8, 100.0, {"factor": 4.0, "fast": 1e9, "original": 64, "slow": 1e8})
    assert abs(f[1] - 100.0 ** -0.25 / 4.0) < 1e-12 and f[0] == 1.0 and abs(amp - 1.1386294361119891) < 1e-12
    w = plain.softmax_with_sink(torch.tensor([0.0, math.log(3.0)], dtype=F64), torch.tensor(math.log(4.0), dtype=F64))
    assert torch.allclose(w, torch.tensor([1 / 8, 3 / 8], dtype=F64))
    y = plain.causal_conv(torch.tensor([[1.0], [2.0], [3.0]], dtype=F64), torch.tensor([[10.0, 1.0]], dtype=F64), torch.tensor([0.5], dtype=F64))
    assert y[:, 0].tolist() == [1.5, 12.5, 23.5]
    # one head, one state, one channel: S halves a token (decay exp(-ln 2)), dt 1 takes B x in, what is read is C S + D x
    one = lambda *a: torch.tensor(a, dtype=F64)
    y = plain.ssd_scan(one(2.0, 4.0).view(2, 1, 1), one(3.0, 5.0).view(2, 1, 1), one(1.0, 10.0).view(2, 1, 1), one(1.0, 1.0).view(2, 1),
                       one(math.log(math.log(2.0))), one(0.25))
    assert torch.allclose(y.flatten(), one(6.0 + 0.5, 10.0 * (3.0 + 20.0) + 1.0))
    n = plain.gated_group_norm(one(3.0, 4.0, 0.0, 5.0).view(1, 4), torch.full((1, 4), 50.0, dtype=F64), one(1.0, 1.0, 1.0, 2.0), 2, 0.0)
    assert torch.allclose(n[0], one(3.0, 4.0, 0.0, 10.0) / one(math.sqrt(12.5), math.sqrt(12.5), 1.0, math.sqrt(12.5)))
    assert plain.run_order(4, {"start": 1, "stop": 3, "times": 2}) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    ff = plain.relu_squared_ff(torch.eye(2, dtype=F64), torch.tensor([[3.0, -2.0]], dtype=F64), torch.ones(1, 1, dtype=F64))
    assert ff[:, 0].tolist() == [9.0, 0.0]

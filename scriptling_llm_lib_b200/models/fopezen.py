"""Layout of the Fopezen decoder: which parts, with which numbers and tensor names.

The embedding is x = `embed`[token] + a vector of sines and cosines of the token's position; nothing else in the model
knows positions but the masks. A layer is x += norm1(mixer(x)) and, where it has a feed-forward, x += norm2(ff(x)): the
sublayers read the stream itself, the norms (RMS, weights stored around zero: `l<i>.norm1`, `.norm2`) stand behind them.

The mixer (`l<i>.mix.*`) is grouped-query softmax attention with biases on its projections (`q.b`, `k.b`, `v.b`), a query/key
norm (`q.norm`, `k.norm`, plain weights), no rotation, a sliding window behind which the sequence's first positions stay
visible, and values that take in a share (`vmix`) of those of the first layer that mixes. Two forms:
`attention`   the norm is per head; one is added to the softmax's denominator (a sink of score 0); the concatenated heads
              are multiplied element by element with sigmoid(`g` x); the output product has a bias too (`o.b`);
`attention_2` the norm is over the whole projection; a plain softmax; no gate, no output bias.

The feed-forward (`l<i>.mlp.up`, `.down`) is dense with the square of relu. The head is the embedding behind `final.norm`.
"""
from __future__ import annotations

from ..config.fopezen import FopezenConfig
from ..config.registry import register_architecture
from ..engine.layout import ModelLayout, sequential_schedule
from ..parts.base import PartSpec
from ..parts.block import LayerSpec
from ..parts.embedding import linear_head

MAX_POSITIONS = 1 << 20      # the family states no longest sequence; the cache's size bounds it
POSITION_BASE = 10000.0      # the family's constant of the position vector's angles


def _norm(cfg: FopezenConfig, name: str) -> PartSpec:
    return PartSpec("rmsnorm", dict(width=cfg.width, eps=cfg.norm_eps, weight_name=name, around_zero=True))


def _mixer(cfg: FopezenConfig, i: int, p: str) -> PartSpec:
    layer = cfg.layers[i]
    m, gated = layer.mixer, layer.type == "attention"
    biases = {n + "_name": f"{p}{n}.b" for n in (("q", "k", "v", "o") if gated else ("q", "k", "v"))}
    value_mix = dict(share_name=p + "vmix", first=i == cfg.first_mixed) if m.v_mix else None
    return PartSpec("attention", dict(
        hidden=cfg.width, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, v_dim=m.vdim, position=None, scale=m.scale,
        window=m.window, keep_first=m.keep_first, biases=biases,
        qk_norm=dict(q_name=p + "q.norm", k_name=p + "k.norm", eps=cfg.norm_eps, per="head" if gated else "projection"),
        sink_value=0.0 if gated else None, gate_name=p + "g" if gated else None, gate_per="element", value_mix=value_mix,
        q_name=p + "q", k_name=p + "k", v_name=p + "v", o_name=p + "o"))


def fopezen_layout(cfg: FopezenConfig) -> ModelLayout:
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"mixer": _mixer(cfg, i, p + "mix."), "mixer_norm": _norm(cfg, p + "norm1")}
        if layer.mlp is not None:
            parts["feed_forward"] = PartSpec("act_feed_forward", dict(hidden=cfg.width, intermediate=layer.mlp.ff, act="relu_squared",
                                                                      up_name=p + "mlp.up", down_name=p + "mlp.down"))
            parts["feed_forward_norm"] = _norm(cfg, p + "norm2")
        layers.append(LayerSpec("post_norm", parts))
    return ModelLayout(
        vocab_size=cfg.vocab, hidden_size=cfg.width, max_positions=MAX_POSITIONS,
        embedding=PartSpec("sinusoid_embedding", dict(vocab=cfg.vocab, width=cfg.width, name="embed", base=POSITION_BASE)),
        layers=tuple(layers), schedule=sequential_schedule(len(layers)), final_norm=_norm(cfg, "final.norm"),
        head=linear_head(cfg.vocab, cfg.width, "embed", tied=True),
        # layers that do not mix have no use for a share that stands in the file all the same
        ignorable_tensors=tuple(f"l{i}.mix.vmix" for i, l in enumerate(cfg.layers) if not l.mixer.v_mix))


register_architecture("Fopezen", FopezenConfig, fopezen_layout)

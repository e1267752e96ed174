"""Layout of the Debusun decoder: which parts, with which numbers and tensor names.

The embedding is x = s `embed`[token] + `bigram`[r], r a hash of (previous token, token) and the table's last row for a
sequence's first token. A layer is x += mixer(norm1(x)); x += ff(norm2(x)) where it has a feed-forward, with RMS norms
(`l<i>.norm1`, `.norm2`, `final.norm`). A run of layers may be gone through several times with the same weights (`loop`):
every appearance has a cache unit or state of its own; before pass t's first layer the stream takes, from the second pass
on, the embedding's output again, and then the vector `loop.step`[t].

The mixer (`l<i>.mix.*`) is one of three. `attention`: grouped-query softmax attention behind a sliding window,
neighbouring pairs of the leading dims turned, queries and keys then divided by their root mean square per head (no
weight). `latent_attention`: direct queries (`q`), keys and values from a cached normed latent (`dkv`, `dkv.norm`, `uk`, `uv`)
with one rotated key part for all heads (frequencies rescaled along a ramp), a sliding window, a stored sink per head
in the softmax's denominator (`sink`), and the concatenated heads multiplied element by element with sigmoid(`g` h).
`mamba2`: a recurrence with one decay per head and token (`in`, `conv`, `conv.b`, `dt_bias`, `A_log`, `D`, `norm`, `o`).

The feed-forward (`l<i>.mlp.up`, `.down`) is dense with the square of relu. The head `head` is a matrix of its own.
"""
from __future__ import annotations

from ..config.debusun import DebusunConfig
from ..config.registry import register_architecture
from ..engine.layout import ModelLayout, looped_schedule, sequential_schedule
from ..parts.base import PartSpec
from ..parts.block import LayerSpec
from ..parts.embedding import linear_head, token_embedding
from ..parts.rotary import YarnScaling

MAX_POSITIONS = 1 << 20      # the family states no longest sequence; the cache's size bounds it


def _norm(cfg: DebusunConfig, name: str) -> PartSpec:
    return PartSpec("rmsnorm", dict(width=cfg.width, eps=cfg.norm_eps, weight_name=name))


def _rotary(rot, width: int) -> PartSpec | None:
    if rot is None:
        return None
    s = rot.scaling
    scaling = YarnScaling(s["factor"], s["original"], s["fast"], s["slow"]) if s is not None else None
    return PartSpec("rotary", dict(head_dim=width, rotary_dim=rot.dims, theta=rot.base, scaling=scaling, pairing="interleaved"))


def _mixer(cfg: DebusunConfig, layer, p: str) -> PartSpec:
    m = layer.mixer
    if layer.type == "attention":
        return PartSpec("attention", dict(
            hidden=cfg.width, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, v_dim=m.vdim, position=_rotary(m.rot, m.dim),
            scale=m.scale, window=m.window, qk_norm=dict(eps=cfg.norm_eps, per="head", after_rotation=True),
            q_name=p + "q", k_name=p + "k", v_name=p + "v", o_name=p + "o"))
    if layer.type == "latent_attention":
        return PartSpec("latent_attention", dict(
            hidden=cfg.width, n_heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, v_dim=m.vdim, kv_rank=m.kv_rank, scale=m.scale,
            position=_rotary(m.rot, m.rot_dim), norm_eps=cfg.norm_eps, window=m.window, sink_name=p + "sink", gate_name=p + "g",
            gate_per="element", q_name=p + "q", uk_name=p + "uk", uv_name=p + "uv", o_name=p + "o", dkv_name=p + "dkv",
            dkv_norm_name=p + "dkv.norm", prompt_kernel="tensor"))
    return PartSpec("mamba2", dict(
        hidden=cfg.width, n_heads=m.heads, head_dim=m.vdim, n_state=m.state, n_groups=m.groups, conv_taps=m.conv,
        norm_groups=m.norm_groups, norm_eps=cfg.norm_eps, in_name=p + "in", conv_name=p + "conv", conv_bias_name=p + "conv.b",
        dt_bias_name=p + "dt_bias", a_log_name=p + "A_log", d_name=p + "D", norm_name=p + "norm", o_name=p + "o"))


def debusun_layout(cfg: DebusunConfig) -> ModelLayout:
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"mixer_norm": _norm(cfg, p + "norm1"), "mixer": _mixer(cfg, layer, p + "mix.")}
        if layer.ff is not None:
            parts["feed_forward_norm"] = _norm(cfg, p + "norm2")
            parts["feed_forward"] = PartSpec("act_feed_forward", dict(hidden=cfg.width, intermediate=layer.ff, act="relu_squared",
                                                                      up_name=p + "mlp.up", down_name=p + "mlp.down"))
        layers.append(LayerSpec("pre_norm_input", parts))
    stream_parts: tuple[PartSpec, ...] = ()
    again = False                   # the embedding's output is added to the stream once more later on
    if cfg.loop is None:
        schedule = sequential_schedule(len(layers))
    else:
        lp, again = cfg.loop, cfg.loop.times > 1
        stream_parts = tuple(PartSpec("pass_vector", dict(width=cfg.width, table_name="loop.step", rows=lp.times, row=t, owns_table=t == 0))
                             for t in range(lp.times)) + (PartSpec("embedding_again"),)
        schedule = looped_schedule(len(layers), lp.start, lp.stop, lp.times,
                                   before_pass=lambda t: (lp.times, t) if t > 0 else (t,))
    if cfg.bigram is None:
        embedding = token_embedding(cfg.vocab, cfg.width, "embed", scale=cfg.embedding_scale, keep_output=again)
    else:
        b = cfg.bigram
        embedding = PartSpec("pair_hash_embedding", dict(vocab=cfg.vocab, width=cfg.width, name="embed", pair_name="bigram",
                                                         buckets=b.buckets, mul_prev=b.mul_prev, mul_cur=b.mul_cur,
                                                         scale=cfg.embedding_scale, keep_output=again))
    return ModelLayout(
        vocab_size=cfg.vocab, hidden_size=cfg.width, max_positions=MAX_POSITIONS, embedding=embedding, layers=tuple(layers),
        schedule=schedule, final_norm=_norm(cfg, "final.norm"), head=linear_head(cfg.vocab, cfg.width, "head"),
        stream_parts=stream_parts)


register_architecture("Debusun", DebusunConfig, debusun_layout)

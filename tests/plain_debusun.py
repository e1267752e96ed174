"""A plain statement of the Debusun decoder in float64: one function per mechanism, whole sequences, explicit
loops, keys and values formed per head and position, the recurrence walked token by token. It shares no code with
the library; the tests compare the library's numbers with these.

`plain_model(raw, W, tokens)` takes the configuration as the dict that config.json holds, the weights as a
dict name -> float64 tensor, and one sequence's token ids; it returns the logits of every position and the
residual stream after every layer run.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_div(x, eps):
    """x over its root mean square (eps under the root), along the last dim."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(v):
    return v * torch.sigmoid(v)


def softplus(v):
    return torch.logaddexp(v, torch.zeros_like(v))


def pair_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table at every position; the table's last row where there is no token before."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + t * mul_cur) % buckets for i, t in enumerate(tokens)]


def embed(tokens, table, scale, pair_table=None, bigram=None):
    x = table[torch.tensor(tokens)] * scale
    if pair_table is not None:
        x = x + pair_table[torch.tensor(pair_rows(tokens, bigram["buckets"], bigram["mul_prev"], bigram["mul_cur"]))]
    return x


def frequencies(dims, base, scaling=None):
    """Angle per position of every pair, and what cos and sin are multiplied by. With a scaling, pairs that turn often
    over the original length keep their pace, slow ones are slowed by the factor, a ramp over the pair index between."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f, 1.0
    where = lambda turns: dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(scaling["fast"])), 0), min(math.ceil(where(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        slow = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(slow * fi / scaling["factor"] + (1.0 - slow) * fi)
    return out, 1.0 + 0.1 * math.log(scaling["factor"])


def rotate(x, dims, base, scaling=None):
    """x [T, heads, d]: row t's neighbouring pairs among the first `dims` entries of every head turn by t * f_i."""
    if dims < 2:
        return x
    f, amp = frequencies(dims, base, scaling)
    out = x.clone()
    for i in range(dims // 2):
        a = torch.arange(x.shape[0], dtype=F64)[:, None] * f[i]
        c, s = torch.cos(a) * amp, torch.sin(a) * amp
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def visible(t, window):
    """First position that position t sees: its own and the window - 1 before it."""
    return 0 if window is None else max(0, t - window + 1)


def softmax_with_sink(scores, sink=None):
    """Weights of the visible keys; a sink adds exp(sink) to the denominator and nothing else."""
    m = scores.max() if sink is None else torch.maximum(scores.max(), sink)
    e = torch.exp(scores - m)
    return e / (e.sum() if sink is None else e.sum() + torch.exp(sink - m))


def _window(m):
    return m["mask"]["size"] if m.get("mask") else None


def attention_mixer(h, W, p, m, eps):
    """Grouped queries behind a window; queries and keys are put on the unit root mean square after they have turned."""
    T, H, G, d, vd = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = (h @ W[p + "q"].T).view(T, H, d), (h @ W[p + "k"].T).view(T, G, d)
    v = (h @ W[p + "v"].T).view(T, G, vd)
    rot = m.get("rot")
    if rot:
        q, k = rotate(q, rot["dims"], rot["base"]), rotate(k, rot["dims"], rot["base"])
    q, k = rms_div(q, eps), rms_div(k, eps)
    out = torch.zeros(T, H, vd, dtype=F64)
    for t in range(T):
        lo = visible(t, _window(m))
        for i in range(H):
            g = i // (H // G)
            out[t, i] = softmax_with_sink((k[lo:t + 1, g] @ q[t, i]) * m["scale"]) @ v[lo:t + 1, g]
    return out.reshape(T, H * vd) @ W[p + "o"].T


def latent_attention_mixer(h, W, p, m, eps):
    """Keys and values from a normed latent, one rotated key part for all heads, a window, a sink per head, a gate per
    output element."""
    T, H, d, r, vd, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m.get("rot")
    q = (h @ W[p + "q"].T).view(T, H, d + r)
    down = h @ W[p + "dkv"].T
    c = rms_div(down[:, :R], eps) * W[p + "dkv.norm"]
    qr, kr = q[:, :, d:], down[:, R:].reshape(T, 1, r)
    if rot:
        qr, kr = (rotate(a, rot["dims"], rot["base"], rot.get("scaling")) for a in (qr, kr))
    ku, vu = (c @ W[p + "uk"].T).view(T, H, d), (c @ W[p + "uv"].T).view(T, H, vd)
    out = torch.zeros(T, H, vd, dtype=F64)
    for t in range(T):
        lo = visible(t, _window(m))
        for i in range(H):
            s = (ku[lo:t + 1, i] @ q[t, i, :d] + kr[lo:t + 1, 0] @ qr[t, i]) * m["scale"]
            out[t, i] = softmax_with_sink(s, W[p + "sink"][i]) @ vu[lo:t + 1, i]
    return (out.reshape(T, H * vd) * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def causal_conv(x, w, b):
    """Every channel's own filter over the rows so far; the last tap is the row's own, rows before the first are zero."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y + b


def ssd_scan(x, B, C, dt, a_log, D):
    """x [T, H, V], B and C [T, G, N], dt [T, H] (after softplus): the state of head i, [N, V], shrinks by one number a
    token and takes dt B x^T in; what is read out is S^T C + D x."""
    T, H, V = x.shape
    G, N = B.shape[1], B.shape[2]
    y = torch.zeros(T, H, V, dtype=F64)
    for i in range(H):
        g = i // (H // G)
        S = torch.zeros(N, V, dtype=F64)
        for t in range(T):
            S = torch.exp(-torch.exp(a_log[i]) * dt[t, i]) * S + dt[t, i] * torch.outer(B[t, g], x[t, i])
            y[t, i] = S.T @ C[t, g] + D[i] * x[t, i]
    return y


def gated_group_norm(y, z, w, groups, eps):
    """y silu(z), then every one of `groups` equal runs of columns over its own root mean square, then the weight."""
    u = y * silu(z)
    return rms_div(u.view(u.shape[0], groups, -1), eps).reshape(u.shape) * w


def mamba2_mixer(h, W, p, m, eps):
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = torch.split(h @ W[p + "in"].T, [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(causal_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    y = ssd_scan(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + W[p + "dt_bias"]), W[p + "A_log"],
                 W[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, W[p + "norm"], m["norm_groups"], eps) @ W[p + "o"].T


def relu_squared_ff(h, up, down):
    return torch.clamp(h @ up.T, min=0.0) ** 2 @ down.T


def run_order(n_layers, loop):
    """(layer, number of the pass it opens or None) for every layer run."""
    if not loop:
        return [(i, None) for i in range(n_layers)]
    a, b = loop["start"], loop["stop"]
    order = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t if i == a else None) for i in range(a, b)]
    return order + [(i, None) for i in range(b, n_layers)]


def plain_model(raw, W, tokens):
    W = {n: w.to(F64) for n, w in W.items()}
    eps = raw["norm"]["eps"]
    emb = raw.get("embedding") or {}
    first = embed(tokens, W["embed"], emb.get("scale", 1.0), W.get("bigram"), emb.get("bigram"))
    x = first
    streams = []
    mixers = {"attention": attention_mixer, "latent_attention": latent_attention_mixer, "mamba2": mamba2_mixer}
    for i, t in run_order(len(raw["layers"]), raw.get("loop")):
        layer, p = raw["layers"][i], f"l{i}."
        if t is not None:
            if t > 0:
                x = x + first
            x = x + W["loop.step"][t]
        x = x + mixers[layer["type"]](rms_div(x, eps) * W[p + "norm1"], W, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + relu_squared_ff(rms_div(x, eps) * W[p + "norm2"], W[p + "mlp.up"], W[p + "mlp.down"])
        streams.append(x.clone())
    return (rms_div(x, eps) * W["final.norm"]) @ W["head"].T, torch.stack(streams)

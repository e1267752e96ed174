"""A plain statement of the Fopezen decoder in float64: one function per mechanism, whole sequences, a query at a
time. It shares no code with the library; the tests compare the library's numbers with these.

`plain_model(raw, W, tokens)` takes the configuration as the dict that config.json holds, the weights as a
dict name -> float64 tensor, and one sequence's token ids; it returns the logits of every position and the
residual stream after every layer. `r` (default: identity) is applied wherever an engine that works in a
narrower format stores an activation, so the same statement serves as the reference of a bfloat16 run.
"""
from __future__ import annotations

import torch

F64 = torch.float64


def same(x):
    return x


def to_bf16(x):
    return x.to(torch.bfloat16).to(F64)


def rms_div(x, eps):
    """x divided by its root mean square (eps inside the root), along the last dim."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def shifted_rms_norm(x, w, eps):
    """RMS norm whose stored weight is the deviation from one."""
    return rms_div(x, eps) * (1.0 + w)


def sinusoid(p, width):
    """The vector a token at position p adds to its embedding: sine at even entries, cosine at odd ones, the
    angle p * 10000^(-2i / width) for the pair (2i, 2i + 1); an odd width ends on a sine."""
    i = torch.arange((width + 1) // 2, dtype=F64)
    angle = p * torch.pow(torch.tensor(10000.0, dtype=F64), -2.0 * i / width)
    out = torch.zeros(2 * i.shape[0], dtype=F64)
    out[0::2], out[1::2] = torch.sin(angle), torch.cos(angle)
    return out[:width]


def embed(tokens, table):
    return torch.stack([table[t] + sinusoid(p, table.shape[1]) for p, t in enumerate(tokens)])


def sees(i, j, size, keep):
    """Whether position i sees position j: a window of `size` positions (None: no window) and the first `keep`."""
    if j > i:
        return False
    return size is None or i - j < size or j < keep


def head_norms(x, w, heads, eps, whole):
    """The query/key norm of one projection [T, heads * d]: over the whole row, or over every head by itself."""
    if whole:
        return rms_div(x, eps) * w
    T = x.shape[0]
    return (rms_div(x.view(T, heads, -1), eps) * w).reshape(T, -1)


def weights_of(scores, plus_one):
    """Softmax of the visible keys' scores; `plus_one`: one more entry of score 0 in the denominator."""
    m = scores.max()
    if plus_one:
        m = torch.maximum(m, torch.zeros((), dtype=F64))
    e = torch.exp(scores - m)
    return e / (e.sum() + (torch.exp(-m) if plus_one else 0.0))


def attend(q, k, v, H, G, scale, size, keep, plus_one):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H * dv]."""
    T = q.shape[0]
    out = torch.zeros((T, H, v.shape[-1]), dtype=F64)
    for i in range(T):
        js = torch.tensor([j for j in range(i + 1) if sees(i, j, size, keep)])
        for h in range(H):
            g = h // (H // G)
            out[i, h] = weights_of((k[js, g] @ q[i, h]) * scale, plus_one) @ v[js, g]
    return out.reshape(T, -1)


def mixed_values(v, first, lam):
    """Values of a layer behind the first value-mixing one: part of its own, part of that layer's."""
    return (1.0 - lam) * v + lam * first


def mixer(h, W, p, m, kind, eps, first_values, r=same):
    """-> (output, this layer's values). `first_values`: those of the first value-mixing layer, or None."""
    H, G, T = m["heads"], m["kv_heads"], h.shape[0]
    q, k, v = (r(h @ W[p + c].T + W[p + c + ".b"]) for c in "qkv")
    whole = kind == "attention_2"
    q = r(head_norms(q, W[p + "q.norm"], H, eps, whole))
    k = r(head_norms(k, W[p + "k.norm"], G, eps, whole))
    if m.get("v_mix") and first_values is not None:
        v = r(mixed_values(v, first_values, W[p + "vmix"]))
    mask = m.get("mask") or {}
    a = r(attend(q.view(T, H, -1), k.view(T, G, -1), v.view(T, G, -1), H, G, m["scale"], mask.get("size"),
                 mask.get("keep_first", 0), plus_one=kind == "attention"))
    if kind == "attention":
        a = r(a * torch.sigmoid(r(h @ W[p + "g"].T)))
    y = a @ W[p + "o"].T
    if kind == "attention":
        y = y + W[p + "o.b"]
    return r(y), v


def feed_forward(h, W, p, r=same):
    u = torch.clamp(h @ W[p + "up"].T, min=0.0)
    return r(r(u * u) @ W[p + "down"].T)


def plain_model(raw, W, tokens, r=same):
    eps = raw["norm"]["eps"]
    x = embed(tokens, W["embed"])
    streams, first = [], None
    for i, layer in enumerate(raw["layers"]):
        p = f"l{i}."
        y, v = mixer(r(x), W, p + "mix.", layer["mixer"], layer["type"], eps, first, r)
        if layer["mixer"].get("v_mix") and first is None:
            first = v
        x = x + shifted_rms_norm(y, W[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + shifted_rms_norm(feed_forward(r(x), W, p + "mlp.", r), W[p + "norm2"], eps)
        streams.append(x)
    logits = r(shifted_rms_norm(x, W["final.norm"], eps)) @ W["embed"].T
    return logits, torch.stack(streams)

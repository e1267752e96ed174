"""The Debusun decoder on the GPU against the plain statement in plain_debusun.py: each mechanism alone, the residual
stream layer by layer, whole prompts against token-by-token decoding and against portions, unequal batches, slots and
pages used again, keys just inside and just outside windows, at page borders and far back, a recurrence that remembers,
the sink, the first tokens, long decoding through several passes, other sizes, greedy generation through the entry point.
Configurations and weights are made here; weights are larger than a trained model's so that every branch moves the logits."""
import json
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_debusun as plain

pytestmark = pytest.mark.gpu

TOL_F32 = 2e-4       # of a row's largest logit
TOL_BF16 = 6e-2
RAMP = {"factor": 4.0, "fast": 8.0, "original": 64, "slow": 1.0}


def attention(heads=4, kv_heads=2, dim=8, vdim=None, scale=0.4, window=20, dims=4, base=300.0):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": dim if vdim is None else vdim}
    if window:
        m["mask"] = {"size": window}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
    return {"type": "attention", "mixer": m}


def latent(heads=3, dim=6, rot_dim=4, vdim=5, kv_rank=10, scale=0.35, window=30, base=200.0, scaling=None):
    m = {"dim": dim, "heads": heads, "kv_rank": kv_rank, "rot_dim": rot_dim, "scale": scale, "vdim": vdim}
    if window:
        m["mask"] = {"size": window}
    if rot_dim >= 2:
        m["rot"] = {"base": base, "dims": rot_dim}
        if scaling is not None:
            m["rot"]["scaling"] = scaling
    return {"type": "latent_attention", "mixer": m}


def mamba2(heads=4, vdim=6, state=8, groups=2, conv=4, norm_groups=2):
    return {"type": "mamba2", "mixer": {"conv": conv, "groups": groups, "heads": heads, "norm_groups": norm_groups, "state": state,
                                        "vdim": vdim}}


def ff(layer, width):
    return dict(layer, mlp={"ff": width, "kind": "dense"})


def config(layers, width=48, vocab=90, eps=1e-6, scale=None, bigram=None, loop=None):
    cfg = {"architecture": "Debusun", "layers": [dict({"mlp": None}, **l) for l in layers], "norm": {"eps": eps}, "vocab": vocab,
           "width": width}
    if scale is not None or bigram is not None:
        cfg["embedding"] = {} if scale is None else {"scale": scale}
        if bigram is not None:
            cfg["embedding"]["bigram"] = {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


# Sizes that differ from one another in every number. A: three kinds, three passes over the two middle layers. B: no pair
# table, no loop, no scale; one group of heads for each head, a convolution of one tap (no state of it), no window, no rotation.
# C: widths that are multiples of nothing, windows shorter than anything, the whole model gone through twice. D: sizes that the
# tensor-core kernels take (bfloat16): the norm over the whole row, folded into the output product, and one taken apart.
CFG_A = config([ff(latent(scaling=RAMP), 24), ff(mamba2(), 20), attention(vdim=12, window=33), ff(attention(2, 1, 16, 16, 0.3, 70, 16), 16)],
               scale=3.0, bigram=(53, 31, 7), loop=(1, 3, 3))
CFG_B = config([ff(mamba2(3, 10, 20, 3, 1, 6), 40), ff(attention(6, 6, 12, 12, 0.25, None, 0), 32),
                ff(latent(5, 12, 6, 10, 20, 0.2, None, 5000.0), 48)], width=96, vocab=130, eps=1e-5)
CFG_C = config([ff(attention(3, 1, 6, 5, 0.6, 3, 2, 30.0), 9), latent(1, 5, 2, 3, 7, 0.6, 1, 10.0, RAMP), ff(mamba2(5, 3, 7, 1, 3, 5), 11),
                attention(5, 5, 3, 2, 1.0, 65, 2, 7.0)], width=50, vocab=61, scale=0.5, bigram=(17, 5, 3), loop=(0, 4, 2))
CFG_D = config([ff(latent(4, 48, 16, 64, 64, 0.12, 100, 10000.0, RAMP), 128), ff(mamba2(4, 64, 64, 1, 4, 1), 96),
                ff(attention(4, 2, 64, 64, 0.3, 130, 32, 10000.0), 128), ff(mamba2(2, 80, 24, 2, 4, 4), 64),
                ff(attention(2, 1, 128, 96, 0.2, 64, 128, 10000.0), 64)], width=256, vocab=200, scale=2.0, bigram=(251, 131, 11),
               loop=(1, 4, 2))


def random_weights(cfg, seed, std=0.25):
    """Weights by tensor name for `cfg`, bfloat16-representable (the folder stores bfloat16)."""
    from scriptling_llm_lib_b200 import models  # noqa: F401
    from scriptling_llm_lib_b200.config.registry import architecture_for
    from scriptling_llm_lib_b200.engine.model import DecoderModel
    arch = architecture_for("Debusun")
    specs = DecoderModel(arch.layout(arch.config_class.from_dict(cfg, "test"))).tensor_specs()
    g = torch.Generator().manual_seed(seed)
    W = {}
    for s in specs:
        t = torch.randn(s.shape, generator=g)
        if s.init == "norm_weight":
            t = 1.0 + 0.2 * t
        elif s.init == "matrix":
            t = t * std * (4.0 / math.sqrt(s.shape[-1]))
        else:
            t = 0.5 * t
        if s.name.endswith("A_log"):
            t = t - 1.5                          # a memory of some tens of tokens
        W[s.name] = t.to(torch.bfloat16)
    for name, size in (("embed", 1.0), ("bigram", 0.5)):
        if name in W:
            W[name] = (torch.randn(W[name].shape, generator=g) * size).to(torch.bfloat16)
    return W


def write_folder(path, cfg, W):
    from scriptling_llm_lib_b200.weights.safetensors_io import write_safetensors
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(path / "model.safetensors", W)
    return path


def ids(n, vocab, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


def engine(folder, dtype="float32", max_tokens=2048, max_seqs=8, **kw):
    from scriptling_llm_lib_b200.engine.step import Engine
    return Engine.from_folder(folder, dtype, max_tokens=max_tokens, max_seqs=max_seqs, **kw)


def run(eng, pieces):
    """Feed one sequence in the given pieces; logits of every position [T, vocab]."""
    from scriptling_llm_lib_b200.engine.step import StepEntry
    seq = eng.open()
    out = []
    for p in pieces:
        out.append(eng.step([StepEntry(seq, list(p), list(range(len(p))))]))
    eng.check_errors()
    seq.close()
    return torch.cat(out).cpu().double()


def cut(tokens, sizes):
    out, at = [], 0
    for s in sizes:
        out.append(tokens[at:at + s])
        at += s
    if at < len(tokens):
        out.append(tokens[at:])
    return [p for p in out if p]


def rel(got, want):
    return float(((got - want).abs().amax(-1) / want.abs().amax(-1).clamp_min(1e-30)).max())


def near(got, want, tol):
    """bfloat16 against the plain statement: heads that are normed after their projection can come out so short that rounding
    turns them, which carries a row in a hundred off; the others stay well within `tol`."""
    err = (got - want).abs().amax(-1) / want.abs().amax(-1).clamp_min(1e-30)
    return float((err > tol).double().mean()) <= 0.01 and float(err.median()) < tol / 8


_PLAIN = {}


def plain_logits(cfg, W, tokens, layers_out=None):
    """The plain statement's logits (kept: several tests ask for the same sequence)."""
    key = (id(W), tuple(tokens))
    if layers_out is None and key in _PLAIN:
        return _PLAIN[key][1]
    logits, streams = plain.plain_model(cfg, W, tokens)
    if layers_out is not None:
        layers_out.extend(streams)
    _PLAIN[key] = (W, logits)
    return logits


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("debusun")
    out = {}
    for name, cfg, seed in (("A", CFG_A, 1), ("B", CFG_B, 2), ("C", CFG_C, 3), ("D", CFG_D, 4)):
        W = random_weights(cfg, seed)
        out[name] = (write_folder(root / name, cfg, W), cfg, W)
    yield out
    _PLAIN.clear()


# --------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_token_by_token_and_portions_equal_the_plain_statement(folders, name):
    folder, cfg, W = folders[name]
    tokens = ids(210, cfg["vocab"], 14)
    want = plain_logits(cfg, W, tokens)
    eng = engine(folder)
    for sizes in ([210], [1] * 210, [2] * 105, [3, 2, 31, 33, 1, 64, 7, 41], [64, 64, 64], [63, 2, 63, 2], [140] + [1] * 70):
        got = run(eng, cut(tokens, sizes))
        assert rel(got, want) < TOL_F32, sizes


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_bfloat16_stays_near_the_plain_statement(folders, name):
    folder, cfg, W = folders[name]
    tokens = ids(210, cfg["vocab"], 14)
    want = plain_logits(cfg, W, tokens)
    eng = engine(folder, "bfloat16")
    for sizes in ([210], [170] + [1] * 40, [64, 3, 70, 2], [2] * 105):
        assert near(run(eng, cut(tokens, sizes)), want, 2 * TOL_BF16), sizes


def test_the_residual_stream_after_every_layer_run(folders):
    from scriptling_llm_lib_b200.engine.step import StepEntry
    from scriptling_llm_lib_b200.parts.norm import take_into_stream
    for name in ("A", "C"):
        folder, cfg, W = folders[name]
        tokens = ids(57, cfg["vocab"], 12)
        want = []
        plain_logits(cfg, W, tokens, layers_out=want)
        eng = engine(folder)
        assert len(eng.layout.schedule) == len(want)
        seq = eng.open()
        arr = np.asarray(tokens, dtype=np.int64)
        eng.cache.reserve([(seq.slot, len(tokens))])
        ctx = eng._context([StepEntry(seq, tokens, [])], arr, [len(tokens)], [0], [])
        x = eng.model.embedding.forward(ctx.token_ids, ctx)
        delta = None
        for i, e in enumerate(eng.layout.schedule):
            for j in e.before:
                delta = eng.model.stream_parts[j].forward(x, delta, ctx)
            delta = eng.model.blocks[e.layer].forward(x, delta, ctx, e.cache_unit, e.writes_cache)
            full = x.clone()                         # what is pending is taken in by the next norm
            take_into_stream(full, delta, ctx)
            assert float((full.double().cpu() - want[i]).abs().max()) < 1e-4 * float(want[i].abs().max()), f"layer run {i}"
        seq.close()


@pytest.mark.parametrize("layer,extra", [
    (attention(3, 3, 8, 8, 0.5, None, 0), {}), (attention(4, 2, 8, 8, 0.5, None, 8, 100.0), {}),
    (attention(4, 1, 8, 12, 0.5, 17, 4, 100.0), {}), (attention(2, 2, 7, 5, 0.5, None, 4, 50.0), {}), (attention(2, 1, 9, 9, 0.5, 5, 0), {}),
    (latent(2, 6, 0, 6, 8, 0.5, None), {}), (latent(3, 4, 6, 5, 9, 0.5, 40, 40.0, RAMP), {}),
    (mamba2(1, 4, 4, 1, 1, 1), {}), (mamba2(3, 8, 6, 1, 4, 1), {}), (mamba2(4, 5, 3, 4, 2, 10), {}), (mamba2(2, 40, 70, 1, 5, 2), {}),
    (ff(attention(1, 1, 4, 4, 1.0, None, 0), 20), {}), (attention(1, 1, 4, 4, 1.0, None, 0), {"bigram": (23, 3, 5)}),
    (attention(1, 1, 4, 4, 1.0, None, 0), {"scale": 5.0}), (attention(1, 1, 4, 4, 1.0, None, 0), {"loop": (0, 1, 1)}),
    (attention(1, 1, 4, 4, 1.0, None, 0), {"loop": (0, 1, 4), "scale": 2.0, "bigram": (11, 2, 3)}),
], ids=["unit-rms", "rotation", "window", "odd-widths", "no-rotation", "latent", "latent-window", "scan-one", "scan", "scan-groups",
        "scan-wide", "dense", "pair-table", "scale", "one-pass", "passes"])
def test_each_mechanism_alone(tmp_path, layer, extra):
    cfg = config([layer], width=32, vocab=50, **extra)
    W = random_weights(cfg, 5, std=0.4)
    folder = write_folder(tmp_path / "m", cfg, W)
    tokens = ids(75, 50, 13)
    want = plain_logits(cfg, W, tokens)
    eng = engine(folder)
    assert rel(run(eng, [tokens]), want) < TOL_F32
    assert rel(run(eng, [tokens[:20]] + [[t] for t in tokens[20:]]), want) < TOL_F32


# --------------------------------------------------------------------------- batches, slots, pages
@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("C", "float32"), ("D", "bfloat16")])
def test_unequal_requests_in_a_batch_equal_each_alone_and_slots_are_used_again(folders, name, dtype):
    from scriptling_llm_lib_b200.engine.step import StepEntry
    folder, cfg, W = folders[name]
    V = cfg["vocab"]
    reqs = [ids(n, V, 20 + i) for i, n in enumerate((70, 3, 139, 1, 40, 200))]
    prompt = [60, 2, 100, 1, 33, 190]
    want = [plain_logits(cfg, W, r) for r in reqs]
    eng = engine(folder, dtype, max_seqs=6, max_tokens=1024)
    tol = TOL_F32 if dtype == "float32" else 2 * TOL_BF16
    for round_ in range(3):                     # the same slots and pages again, after other requests held them
        seqs = [eng.open() for _ in reqs]
        out = eng.step([StepEntry(s, r[:p], list(range(p))) for s, r, p in zip(seqs, reqs, prompt)]).cpu().double()
        got, at = [[] for _ in reqs], 0
        for i, p in enumerate(prompt):
            got[i].append(out[at:at + p])
            at += p
        pos = list(prompt)
        live = [i for i in range(len(reqs)) if pos[i] < len(reqs[i])]
        for i in range(len(reqs)):
            if i not in live:
                seqs[i].close()
        while live:
            out = eng.step([StepEntry(seqs[i], [reqs[i][pos[i]]], [0]) for i in live]).cpu().double()
            for j, i in enumerate(live):
                got[i].append(out[j:j + 1])
                pos[i] += 1
                if pos[i] == len(reqs[i]):
                    seqs[i].close()
            live = [i for i in live if pos[i] < len(reqs[i])]
        for i in range(len(reqs)):
            assert rel(torch.cat(got[i]), want[i]) < tol, (round_, i)
        reqs, prompt, want = reqs[::-1], prompt[::-1], want[::-1]
    assert eng.cache.slots.n_held == 0 and all(g.pool.n_held == 0 for g in eng.cache.groups)


def test_the_first_tokens_of_a_sequence(folders):
    for name in ("A", "B", "C"):
        folder, cfg, W = folders[name]
        eng = engine(folder)
        for n in (1, 2, 3, 4, 5, 6):
            tokens = ids(n, cfg["vocab"], 30 + n)
            want = plain_logits(cfg, W, tokens)
            assert rel(run(eng, [tokens]), want) < TOL_F32
            assert rel(run(eng, [[t] for t in tokens]), want) < TOL_F32


def test_a_slot_used_again_starts_from_nothing(folders):
    """The previous token, the convolution's inputs and the recurrence's state of the sequence that held the slot before must
    not leak; a portion's first row must find what the portion before it left."""
    folder, cfg, W = folders["A"]
    for dtype, tol in (("float32", TOL_F32), ("bfloat16", 2 * TOL_BF16)):
        eng = engine(folder, dtype, max_seqs=1)
        a, b = ids(40, cfg["vocab"], 50), ids(33, cfg["vocab"], 51)
        for tokens in (a, b, a):
            assert rel(run(eng, cut(tokens, [11, 1, 1, 9])), plain_logits(cfg, W, tokens)) < tol


def test_long_decoding_through_all_passes_gives_pages_back(folders):
    from scriptling_llm_lib_b200.engine.step import StepEntry
    folder, cfg, W = folders["A"]
    tokens = ids(300, cfg["vocab"], 15)
    want = plain_logits(cfg, W, tokens)
    for dtype in ("float32", "bfloat16"):
        eng = engine(folder, dtype, max_tokens=1024)
        seq = eng.open()
        got = [eng.step([StepEntry(seq, tokens[:5], list(range(5)))])]
        for t in tokens[5:]:
            got.append(eng.step([StepEntry(seq, [t], [0])]))
        assert rel(torch.cat(got).cpu().double(), want) < (TOL_F32 if dtype == "float32" else 2 * TOL_BF16)
        for g in eng.cache.groups:                       # a window's pages and no more are held
            assert sum(p >= 0 for p in g.pages[seq.slot]) <= g.need.pages_seen() < 5
        seq.close()


# --------------------------------------------------------------------------- windows' edges, page borders, far memory, the sink
def light_channel(W, loud=39):
    """Embedding channels by hand: the token `loud` lights channel 0, every token carries a constant in channel 1."""
    W["embed"][:, 0] = 0.0
    W["embed"][loud, 0] = 8.0
    W["embed"][:, 1] = 2.0
    W["l0.norm1"][0], W["l0.norm1"][1] = 1.0, 1.0


def loud_attention(tmp_path, window, dim=8, vdim=8, heads=2, kv_heads=1, dims=0):
    """One attention layer whose queries all look for one token (the last id). Heads are normed, so a direction is what counts:
    that token's key lies along dim 0, every query too, other keys have nothing there. With a rotation dim 0 stays behind it."""
    cfg = config([attention(heads, kv_heads, dim, vdim, 10.0 / dim, window, dims, 100.0)], width=32, vocab=40)
    W = random_weights(cfg, 7, std=0.3)
    light_channel(W)
    at = dims                                       # the first dim that does not turn
    W["l0.mix.k"][at, :] = 0.0
    W["l0.mix.k"][at, 0] = 20.0
    for h in range(heads):
        W["l0.mix.q"][h * dim + at, :] = 0.0
        W["l0.mix.q"][h * dim + at, 1] = 30.0
    return write_folder(tmp_path / f"loud{window}_{dim}_{vdim}_{dims}", cfg, W), cfg, W


def loud_latent(tmp_path, window, dim=4, rot_dim=4, vdim=6, rank=8, heads=2, sink=0.0):
    """The same through the cached latent: the shared key part's first dim reads the loud channel (no rotation here), every
    head's first rotated query dim reads the constant."""
    layer = latent(heads, dim, rot_dim, vdim, rank, 1.0, window)
    del layer["mixer"]["rot"]
    cfg = config([layer], width=32, vocab=40)
    W = random_weights(cfg, 8, std=0.3)
    light_channel(W)
    W["l0.mix.dkv"][rank, :] = 0.0
    W["l0.mix.dkv"][rank, 0] = 3.0
    for h in range(heads):
        W["l0.mix.q"][h * (dim + rot_dim) + dim, :] = 0.0
        W["l0.mix.q"][h * (dim + rot_dim) + dim, 1] = 1.5
    W["l0.mix.uk"] *= 0.1                            # the unrotated part stays quiet
    W["l0.mix.sink"].fill_(sink)
    return write_folder(tmp_path / f"loudlatent{window}_{dim}_{rot_dim}_{vdim}", cfg, W), cfg, W


LOUD = [(loud_attention, 40, {}, "float32"), (loud_attention, 64, dict(dim=12, vdim=7, dims=4), "float32"),
        (loud_attention, 65, dict(dim=9, vdim=9), "float32"), (loud_attention, 63, dict(dim=64, vdim=64, dims=32), "bfloat16"),
        (loud_attention, 100, dict(dim=128, vdim=64, heads=4), "bfloat16"), (loud_attention, 70, dict(dim=192, vdim=48), "bfloat16"),
        (loud_latent, 40, {}, "float32"), (loud_latent, 64, dict(dim=5, rot_dim=3, vdim=7, rank=9), "float32"),
        (loud_latent, 100, dict(dim=48, rot_dim=16, vdim=64, rank=64), "bfloat16"),
        (loud_latent, 65, dict(dim=128, rot_dim=32, vdim=40, rank=96), "bfloat16")]


@pytest.mark.parametrize("make,window,kw,dtype", LOUD, ids=[f"{m.__name__}-{w}-{'-'.join(map(str, k.values()))}" for m, w, k, _ in LOUD])
def test_a_loud_key_just_inside_and_just_outside_the_window(tmp_path, make, window, kw, dtype):
    folder, cfg, W = make(tmp_path, window, **kw)
    eng = engine(folder, dtype)
    tol = TOL_F32 if dtype == "float32" else TOL_BF16
    base = ids(200, 39, 16)                          # never the loud token
    other = plain_logits(cfg, W, base)
    for p in (0, 1, 62, 63, 64, 95):
        tokens = list(base)
        tokens[p] = 39
        want = plain_logits(cfg, W, tokens)
        last = p + window - 1                        # the last position that sees it
        assert rel(want[last:last + 1], other[last:last + 1]) > 0.1
        assert rel(want[last + 1:], other[last + 1:]) < 1e-9
        assert rel(run(eng, [tokens]), want) < tol
        for first in (last - 1, last, last + 1):     # decoding starts around the edge
            assert rel(run(eng, [tokens[:first]] + [[t] for t in tokens[first:last + 6]]), want[:last + 6]) < tol
        assert rel(run(eng, cut(tokens, [63, 2, 64, 41])), want) < tol
        assert rel(run(eng, cut(tokens, [last, 2])), want) < tol


def test_a_far_key_without_a_window(tmp_path):
    for make in (loud_attention, loud_latent):
        folder, cfg, W = make(tmp_path, None)
        eng = engine(folder)
        base = ids(200, 39, 16)
        other = plain_logits(cfg, W, base)
        for p in (0, 63, 64, 150):
            tokens = list(base)
            tokens[p] = 39
            want = plain_logits(cfg, W, tokens)
            assert rel(want[190:], other[190:]) > 100 * TOL_F32
            assert rel(run(eng, [tokens]), want) < TOL_F32
            assert rel(run(eng, [tokens[:170]] + [[t] for t in tokens[170:]]), want) < TOL_F32


def test_the_sink_takes_its_share_once(tmp_path):
    """A large sink on one head empties that head's output whatever the number of keys or the way they are split; a sink
    that is left out, or counted once per split, or scaled, shows."""
    for kw, dtype, tol in (({}, "float32", TOL_F32), (dict(dim=48, rot_dim=16, vdim=64, rank=64), "bfloat16", TOL_BF16)):
        folder, cfg, W = loud_latent(tmp_path, 150, heads=4, **kw)
        tokens = ids(300, 39, 18)
        quiet = plain_logits(cfg, W, tokens)
        W["l0.mix.sink"][0], W["l0.mix.sink"][1], W["l0.mix.sink"][3] = 6.0, -3.0, 3.5
        _PLAIN.clear()
        folder = write_folder(tmp_path / ("sink_on" + dtype), cfg, W)
        want = plain_logits(cfg, W, tokens)
        assert rel(want, quiet) > 0.1
        eng = engine(folder, dtype)
        assert rel(run(eng, [tokens]), want) < tol
        assert rel(run(eng, [tokens[:250]] + [[t] for t in tokens[250:]]), want) < tol     # a decode step's keys are split over blocks
        assert rel(run(eng, cut(tokens, [130, 100])), want) < tol


def long_memory(tmp_path, heads=2, vdim=4, state=4, taps=4):
    """A recurrence that hardly forgets (decays next to one): its first token shows hundreds of rows later."""
    cfg = config([mamba2(heads, vdim, state, 1, taps, 1)], width=32, vocab=40)
    W = random_weights(cfg, 9, std=0.4)
    light_channel(W)
    inner, N = heads * vdim, state
    W["l0.mix.A_log"].fill_(-9.0)
    W["l0.mix.in"][inner:2 * inner, 0] = 40.0        # the loud token's input is large; everybody reads it out the same way
    W["l0.mix.in"][2 * inner:2 * inner + N, 1] = 2.0
    W["l0.mix.in"][2 * inner + N:2 * inner + 2 * N, 1] = 2.0
    return write_folder(tmp_path / f"memory{vdim}_{state}", cfg, W), cfg, W


@pytest.mark.parametrize("kw,dtype", [({}, "float32"), (dict(heads=2, vdim=64, state=32), "bfloat16"), (dict(heads=1, vdim=20, state=24), "bfloat16")])
def test_the_recurrence_remembers_across_portions_and_chunks(tmp_path, kw, dtype):
    folder, cfg, W = long_memory(tmp_path, **kw)
    eng = engine(folder, dtype)
    tol = TOL_F32 if dtype == "float32" else TOL_BF16
    base = ids(420, 39, 16)
    other = plain_logits(cfg, W, base)
    for p in (0, 63, 127, 128):
        tokens = list(base)
        tokens[p] = 39
        want = plain_logits(cfg, W, tokens)
        assert rel(want[400:], other[400:]) > 0.09
        assert rel(run(eng, [tokens]), want) < tol
        assert rel(run(eng, cut(tokens, [128, 127, 2, 65, 1, 1])), want) < tol
        assert rel(run(eng, [tokens[:390]] + [[t] for t in tokens[390:]]), want) < tol


# --------------------------------------------------------------------------- kernels by themselves
def _scan_case(dtype, H, G, V, N, lens, seed, a_shift=0.0, dt_size=1.0):
    g = torch.Generator().manual_seed(seed)
    T, B = sum(lens), len(lens)
    xbc = torch.randn(T, H * V + 2 * G * N, generator=g).to(dtype)
    dt = (torch.randn(T, H, generator=g) * dt_size).to(dtype)
    z = torch.randn(T, H * V, generator=g).to(dtype)
    dt_bias, a_log, dskip = torch.randn(H, generator=g), torch.randn(H, generator=g) + a_shift, torch.randn(H, generator=g)
    state = torch.randn(B + 2, H, N, V, generator=g)
    slots = torch.randperm(B + 2, generator=g)[:B].to(torch.int32)
    return xbc, dt, z, dt_bias, a_log, dskip, state, slots


def _scan_plain(xbc, dt, z, dt_bias, a_log, dskip, S0, H, G, V, N):
    """The recurrence of one sequence from a given state, in float64: (y silu(z), last state)."""
    x, Bm, Cm = torch.split(xbc.double(), [H * V, G * N, G * N], dim=1)
    d = plain.softplus(dt.double() + dt_bias.double())
    S, out = S0.double().clone(), torch.zeros(xbc.shape[0], H, V, dtype=torch.float64)
    for t in range(xbc.shape[0]):
        for h in range(H):
            b, c = Bm[t].view(G, N)[h // (H // G)], Cm[t].view(G, N)[h // (H // G)]
            S[h] = torch.exp(-torch.exp(a_log[h].double()) * d[t, h]) * S[h] + d[t, h] * torch.outer(b, x[t].view(H, V)[h])
            out[t, h] = S[h].T @ c + dskip[h].double() * x[t].view(H, V)[h]
    return out.view(-1, H * V) * plain.silu(z.double()), S


@pytest.mark.parametrize("dtype,H,G,V,N,lens,kw", [
    (torch.float32, 3, 1, 5, 7, (1, 20, 3), {}), (torch.float32, 4, 2, 40, 36, (33, 2), {}), (torch.float32, 2, 2, 33, 130, (17,), {}),
    (torch.bfloat16, 2, 1, 64, 128, (130, 1, 300, 128), {}), (torch.bfloat16, 4, 2, 48, 16, (256, 5), {}),
    (torch.bfloat16, 2, 2, 7, 9, (129, 64), {}), (torch.bfloat16, 3, 3, 72, 40, (70, 127), {}), (torch.bfloat16, 2, 1, 130, 200, (140,), {}),
    (torch.bfloat16, 2, 1, 32, 32, (300,), dict(a_shift=4.0, dt_size=6.0)), (torch.bfloat16, 2, 1, 16, 16, (290,), dict(a_shift=-8.0)),
], ids=str)
def test_the_recurrence_walked_and_in_chunks(dtype, H, G, V, N, lens, kw):
    """Against float64 from states that are not zero, on slots out of order: sizes off every step, decays from none to total (a
    chunk's sum of logarithms grows into the thousands). bfloat16 inputs are exact in the products, and what is float enters
    them in three parts, so that states must agree to float accuracy."""
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    k = KernelSet(dtype).ssd
    xbc, dt, z, dt_bias, a_log, dskip, state, slots = _scan_case(dtype, H, G, V, N, lens, 3, **kw)
    starts = np.concatenate([[0], np.cumsum(lens)])
    ctx = SimpleNamespace(n_seqs=len(lens), max_new=max(lens), seq_start=torch.tensor(starts, dtype=torch.int32).cuda(), slots=slots.cuda())
    want, states = [], state.double().clone()
    for b, s in enumerate(slots.tolist()):
        i, j = starts[b], starts[b + 1]
        y, states[s] = _scan_plain(xbc[i:j], dt[i:j], z[i:j], dt_bias, a_log, dskip, state[s], H, G, V, N)
        want.append(y)
    want = torch.cat(want)
    dev = lambda t: t.cuda().contiguous()            # noqa: E731
    wide = torch.zeros(xbc.shape[0], 8 + xbc.shape[1] + (-xbc.shape[1] % 8), dtype=dtype, device="cuda")      # column slices of one buffer
    wide[:, 8:8 + xbc.shape[1]] = xbc.cuda()
    w = torch.rand(H * V, generator=torch.Generator().manual_seed(5)) + 0.5
    for chunked in ((False, True) if dtype == torch.bfloat16 else (False,)):
        for weight in (None, w.cuda()):
            st = dev(state)
            out = torch.full((sum(lens), H * V), float("nan"), dtype=dtype, device="cuda")
            sq = k.scan(wide[:, 8:8 + xbc.shape[1]], dev(dt), dev(dt_bias), dev(a_log), dev(dskip), dev(z), st, ctx, out, H, G, V, N,
                        weight=weight, chunked=chunked)
            scale = float(want.abs().max())
            ref = want if weight is None else want * w.double()
            assert float((out.cpu().double() - ref).abs().max()) < (1e-5 if dtype == torch.float32 else 6e-3) * scale * 1.5
            assert float((st.cpu().double() - states).abs().max()) < 1e-5 * float(states.abs().max())
            if weight is not None:
                assert float((sq.sum(0).cpu().double() / (want * want).sum(-1) - 1.0).abs().max()) < 1e-4


@pytest.mark.parametrize("taps,C", [(2, 12), (3, 520), (4, 64), (4, 516)])
def test_the_convolution_over_many_rows(taps, C):
    """The kernel for steps of many rows: sequences that begin and end inside a thread's rows, runs shorter than the filter, past
    inputs out of the state, bias, SiLU, and the state afterwards."""
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    g = torch.Generator().manual_seed(12)
    lens = (1, 2, 250, 3, 8, 37)
    starts = np.concatenate([[0], np.cumsum(lens)])
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 3e-2)):
        x, w, b = torch.randn(sum(lens), C, generator=g).to(dtype), torch.randn(C, taps, generator=g).to(dtype), torch.randn(C, generator=g).to(dtype)
        state, slots = torch.randn(8, taps - 1, C, generator=g), [5, 0, 7, 2, 3, 1]
        ctx = SimpleNamespace(n_seqs=len(lens), seq_start=torch.tensor(starts, dtype=torch.int32).cuda(), slots=torch.tensor(slots, dtype=torch.int32).cuda(),
                              tok_seq=torch.repeat_interleave(torch.arange(len(lens)), torch.tensor(lens)).to(torch.int32).cuda())
        st, y = state.clone().cuda(), torch.full(x.shape, float("nan"), dtype=dtype, device="cuda")
        KernelSet(dtype).seq.causal_conv(x.cuda(), w.cuda(), st, ctx, y, taps, out_bias=b.cuda(), act="silu")
        for i, slot in enumerate(slots):
            rows = torch.cat([state[slot].double(), x[starts[i]:starts[i + 1]].double()])
            want = plain.silu(plain.causal_conv(rows, w.double(), b.double()))[taps - 1:]
            assert float((y[starts[i]:starts[i + 1]].cpu().double() - want).abs().max()) < tol * 4, (i, dtype)
            assert float((st[slot].cpu().double() - rows[-(taps - 1):]).abs().max()) < 1e-6


def test_the_norm_over_runs_of_columns():
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    g = torch.Generator().manual_seed(6)
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        for W, groups in ((30, 1), (30, 3), (64, 16), (768, 2), (1000, 8), (12, 12)):
            u, w = torch.randn(9, W, generator=g).to(dtype), torch.randn(W, generator=g)
            want = plain.rms_div(u.double().view(9, groups, -1), 1e-3).reshape(9, W) * w.double()
            y = u.clone().cuda()
            KernelSet(dtype).ssd.group_norm(y, w.cuda(), y, groups, 1e-3)
            assert float((y.cpu().double() - want).abs().max()) < tol * 3, (W, groups)


@pytest.mark.parametrize("H,G,hd,vd,rot,interleaved", [(3, 1, 8, 8, 8, True), (2, 2, 128, 64, 32, True), (4, 2, 96, 96, 96, True), (5, 1, 7, 3, 4, True),
                                                       (2, 1, 16, 16, 8, False), (3, 3, 12, 20, 0, True), (2, 1, 9, 9, 0, True), (1, 1, 256, 128, 64, True)])
def test_heads_are_normed_once_they_have_turned(H, G, hd, vd, rot, interleaved):
    """Also with a rotation that stretches (cos and sin times an amplitude): the norm sees what came out."""
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    g = torch.Generator().manual_seed(10)
    T, eps = 6, 0.05
    pos = [0, 1, 63, 64, 65, 70]
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        c = torch.randn(T, (H + G) * hd + G * vd, generator=g).to(dtype)
        ang = torch.rand(80, max(rot // 2, 1), generator=g, dtype=torch.float64) * 6.0
        cs = torch.stack([torch.cos(ang), torch.sin(ang)], -1) * 1.5
        q = torch.empty((T, H * hd), dtype=dtype, device="cuda")
        kp = torch.zeros(3, G, 64, hd, dtype=dtype, device="cuda")
        vp = torch.zeros(3, G, 64, vd, dtype=dtype, device="cuda")
        KernelSet(dtype).gate.qk_norm_store(
            c.cuda(), q, torch.tensor(pos, dtype=torch.int32).cuda(), torch.zeros(T, dtype=torch.int32).cuda(),
            torch.tensor([[2, 0]], dtype=torch.int32).cuda(), cs.float().contiguous().cuda() if rot else None, kp, vp, H, G, hd, vd, rot,
            interleaved, None, None, eps, per_head=True, norm_after=True)
        heads = c[:, :(H + G) * hd].double().view(T, H + G, hd).clone()
        for t, p in enumerate(pos):
            for i in range(rot // 2):
                a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + rot // 2)
                u, v = heads[t, :, a].clone(), heads[t, :, b].clone()
                co, si = cs[p, i, 0].float().double(), cs[p, i, 1].float().double()
                heads[t, :, a], heads[t, :, b] = u * co - v * si, v * co + u * si
        heads = plain.rms_div(heads, eps)
        assert float((q.cpu().double().view(T, H, hd) - heads[:, :H]).abs().max()) < tol * 2
        for t, p in enumerate(pos):
            page = (2, 0)[p // 64]
            assert float((kp[page, :, p % 64].cpu().double() - heads[t, H:]).abs().max()) < tol * 2
            assert torch.equal(vp[page, :, p % 64].cpu(), c[t, (H + G) * hd:].view(G, vd))


def test_the_embedding_scales_its_row_and_keeps_a_copy():
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    g = torch.Generator().manual_seed(11)
    ks = KernelSet(torch.float32)
    table, pair = torch.randn(20, 10, generator=g), torch.randn(8, 10, generator=g)
    tok = torch.tensor([3, 19, 3], dtype=torch.int32).cuda()
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    out, copy = torch.empty((3, 10), device="cuda"), torch.empty((3, 10), device="cuda")
    ks.embed_rows(tok, table.cuda(), out, err, scale=2.5, copy=copy)
    assert torch.allclose(out.cpu(), table[[3, 19, 3]] * 2.5) and torch.equal(out, copy)
    ctx = SimpleNamespace(tok_pos=torch.tensor([0, 1, 2], dtype=torch.int32).cuda(), tok_seq=torch.zeros(3, dtype=torch.int32).cuda(),
                          seq_start=torch.tensor([0, 3], dtype=torch.int32).cuda(), slots=torch.zeros(1, dtype=torch.int32).cuda())
    ks.embed_pair_rows(tok, ctx, table.cuda(), pair.cuda(), 7, 2, 3, torch.zeros(2, dtype=torch.int32).cuda(), out, err, scale=2.5, copy=copy)
    rows = [7, (3 * 2 + 19 * 3) % 7, (19 * 2 + 3 * 3) % 7]
    assert torch.allclose(out.cpu(), table[[3, 19, 3]] * 2.5 + pair[rows]) and torch.equal(out, copy) and int(err) == 0


# --------------------------------------------------------------------------- the entry point
def test_greedy_generation_through_the_entry_point(folders):
    from scriptling_llm_lib_b200 import llm
    folder, cfg, W = folders["A"]
    prompt = ids(41, cfg["vocab"], 19)
    for dtype in ("float32", "bfloat16"):
        out = llm.generate(str(folder), prompt, max_tokens=20, strategy="greedy", dtype=dtype)
        assert len(out) == 20
        lg = plain_logits(cfg, W, prompt + list(out))
        for i, t in enumerate(out):
            row = lg[len(prompt) - 1 + i]
            top2 = row.topk(2).values
            if dtype == "float32" or float(top2[0] - top2[1]) > 0.2 * float(row.abs().max()):
                assert int(row.argmax()) == t
        llm.unload()


def test_a_batch_of_unequal_prompts_generates_what_each_alone_does(folders):
    from scriptling_llm_lib_b200 import llm
    folder, cfg, W = folders["C"]
    prompts = [ids(n, cfg["vocab"], 60 + n) for n in (3, 70, 1, 18)]
    alone = [llm.generate(str(folder), p, max_tokens=12, strategy="greedy", dtype="float32") for p in prompts]
    together = llm.generate(str(folder), prompts, max_tokens=12, strategy="greedy", dtype="float32")
    assert together == alone
    llm.unload()


def test_random_weights_mode_and_the_command_line(tmp_path):
    import subprocess
    import sys
    from pathlib import Path
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(CFG_B))
    eng = engine(f"random:{cfg_path}:3", "bfloat16")
    got = run(eng, [ids(40, CFG_B["vocab"], 1)])
    assert torch.isfinite(got).all() and float(got.abs().max()) > 0
    root = Path(__file__).resolve().parent.parent
    r = subprocess.run([sys.executable, "-m", "scriptling_llm_lib_b200", "-model", f"random:{cfg_path}:3", "-prompt", "1,2,3",
                        "-tokens", "4"], cwd=root, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr


def test_trace_replay_writes_the_logits_of_the_wanted_places(folders, tmp_path):
    import subprocess
    import sys
    from pathlib import Path
    folder, cfg, W = folders["C"]
    V = cfg["vocab"]
    a, b = ids(30, V, 40), ids(9, V, 41)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:25], "want": [0, 24]}, {"id": "b", "tokens": b[:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[25:26], "want": [0]}, {"id": "b", "tokens": b[8:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[26:27], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[27:], "want": [2]}], "end": ["a"]}]
    root = Path(__file__).resolve().parent.parent
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = plain_logits(cfg, W, a), plain_logits(cfg, W, b)
    read = lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V).copy()).double()    # noqa: E731
    assert rel(read(0), wa[[0, 24]]) < TOL_F32
    assert rel(read(1), torch.stack([wa[25], wb[8]])) < TOL_F32
    assert not (out / "2.f32").exists()
    assert rel(read(3), wa[29:30]) < TOL_F32

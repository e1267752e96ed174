"""The Fopezen decoder on the GPU against the plain statement in plain_fopezen.py: each mechanism alone, the residual stream
layer by layer, whole prompts against token-by-token decoding and against portions, unequal batches, slots and pages used
again, keys far back, at page borders and on either side of a window's edge and of the last kept position, the first tokens,
long decoding, other sizes, the kernels by themselves, greedy generation through the entry point. Configurations and weights
are made here; weights are larger than a trained model's so that every branch moves the logits."""
import json
import math

import numpy as np
import pytest
import torch

import plain_fopezen as plain

pytestmark = pytest.mark.gpu

TOL_F32 = 1e-4       # of a row's largest logit
TOL_BF16 = 4e-2


def layer(kind="attention", heads=4, kv_heads=2, dim=8, vdim=6, scale=0.4, window=None, keep=0, v_mix=False, ff=20):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "v_mix": v_mix, "vdim": vdim}
    if window is not None:
        m["mask"] = {"keep_first": keep, "size": window}
    return {"type": kind, "mixer": m, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


def config(layers, width=48, vocab=90, eps=1e-6):
    return {"architecture": "Fopezen", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# Sizes that differ from one another in every number. A: both forms, a layer without a window, one without a feed-forward, one
# that does not mix; windows shorter than a page. B: widths that are multiples of nothing, one key/value head, more positions
# kept than the window is long, one head a group. C: heads of 64 and 128 (the tcgen05 prompt kernels), kept positions past a
# page. D: widths in multiples of 8 that differ (the mma.sync kernels), twelve heads a group, wide keys.
CFG_A = config([layer("attention_2", 4, 2, 12, 8, 0.3, 20, 3, True), layer("attention", 6, 2, 10, 8, 0.4, 37, 5, True, None),
                layer("attention", 2, 1, 4, 12, 0.7), layer("attention_2", 3, 1, 8, 16, 0.35, 11, 0, True, 32)], eps=1e-5)
CFG_B = config([layer("attention", 3, 1, 5, 7, 0.6, 9, 14, True, 13), layer("attention_2", 2, 2, 7, 3, 0.5, 70, 66),
                layer("attention", 7, 7, 3, 1, 0.9, 5, 1, True, 6)], width=35, vocab=61)
CFG_C = config([layer("attention_2", 4, 2, 64, 64, 0.15, 100, 70, True, 96), layer("attention", 4, 2, 64, 64, 0.2, 65, 4, True, 64),
                layer("attention", 2, 1, 128, 128, 0.12, 130, 129, True), layer("attention_2", 3, 1, 128, 128, 0.1, None, 0, False, 32),
                layer("attention", 3, 3, 128, 128, 0.1, 30, 12)], width=128, vocab=200)
CFG_D = config([layer("attention", 12, 1, 72, 48, 0.12, 64, 130, True, 48), layer("attention_2", 4, 2, 160, 24, 0.09, 90, 10, True, 40),
                layer("attention", 6, 3, 24, 16, 0.25, 33, 1, True, 24), layer("attention_2", 10, 5, 40, 104, 0.2, 128, 64, False, None)],
               width=80, vocab=150)
ALL = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}


def random_weights(cfg, seed, std=0.25):
    """Weights by tensor name for `cfg`, bfloat16-representable (the folder stores bfloat16)."""
    from scriptling_llm_lib_b200 import models  # noqa: F401
    from scriptling_llm_lib_b200.config.registry import architecture_for
    from scriptling_llm_lib_b200.engine.model import DecoderModel
    arch = architecture_for("Fopezen")
    specs = DecoderModel(arch.layout(arch.config_class.from_dict(cfg, "test"))).tensor_specs()
    g = torch.Generator().manual_seed(seed)
    W = {}
    for s in specs:
        t = torch.randn(s.shape, generator=g)
        if s.init == "norm_weight":
            t = 1.0 + 0.2 * t
        elif s.init == "norm_shift":
            t = 0.2 * t
        elif s.init == "share":
            t = 0.45 + 0.1 * t
        elif s.init == "matrix":
            t = t * std * (4.0 / math.sqrt(s.shape[-1]))
        else:
            t = 0.5 * t
        W[s.name] = t.to(torch.bfloat16)
    W["embed"] = (0.7 * torch.randn(W["embed"].shape, generator=g)).to(torch.bfloat16)
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
    out = [eng.step([StepEntry(seq, list(p), list(range(len(p))))]) for p in pieces]
    eng.check_errors()
    seq.close()
    return torch.cat(out).cpu().double()


def cut(tokens, sizes):
    out, at = [], 0
    for s in sizes:
        out.append(tokens[at:at + s])
        at += s
    return [p for p in out + [tokens[at:]] if p]


def rel(got, want):
    return float(((got - want).abs().amax(-1) / want.abs().amax(-1).clamp_min(1e-30)).max())


def plain_logits(cfg, W, tokens, rounded=False):
    return plain.plain_model(cfg, {n: t.double() for n, t in W.items()}, tokens, plain.to_bf16 if rounded else plain.same)[0]


def tol_of(dtype):
    return TOL_F32 if dtype == "float32" else TOL_BF16


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("fopezen")
    out = {}
    for i, (name, cfg) in enumerate(ALL.items()):
        W = random_weights(cfg, i + 1)
        out[name] = (write_folder(root / name, cfg, W), cfg, W)
    return out


# --------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ALL))
def test_a_whole_prompt_equals_the_plain_statement(folders, name, dtype):
    folder, cfg, W = folders[name]
    tokens = ids(231, cfg["vocab"], 11)
    want = plain_logits(cfg, W, tokens, dtype == "bfloat16")
    assert rel(run(engine(folder, dtype), [tokens]), want) < tol_of(dtype)


def test_the_residual_stream_after_every_layer(folders):
    from scriptling_llm_lib_b200.engine.step import StepEntry
    from scriptling_llm_lib_b200.parts.norm import take_into_stream
    for name in ("A", "B"):
        folder, cfg, W = folders[name]
        tokens = ids(57, cfg["vocab"], 12)
        want = plain.plain_model(cfg, {n: t.double() for n, t in W.items()}, tokens)[1]
        eng = engine(folder)
        seq = eng.open()
        eng.cache.reserve([(seq.slot, len(tokens))])
        ctx = eng._context([StepEntry(seq, tokens, [])], np.asarray(tokens, dtype=np.int64), [len(tokens)], [0], [])
        x, delta = eng.model.embedding.forward(ctx.token_ids, ctx), None
        for i, e in enumerate(eng.layout.schedule):
            delta = eng.model.blocks[e.layer].forward(x, delta, ctx, e.cache_unit, e.writes_cache)
            full = x.clone()                         # what is pending is taken in by the next reader
            take_into_stream(full, delta, ctx)
            assert float((full.double().cpu() - want[i]).abs().max()) < 1e-5 * float(want[i].abs().max()), f"layer {i}"
        seq.close()


@pytest.mark.parametrize("one", [
    layer("attention"), layer("attention_2"), layer("attention", ff=None), layer("attention_2", 1, 1, 16, 4, 0.3, ff=None),
    layer("attention", 5, 5, 6, 6, 0.5, 7, 0), layer("attention_2", 4, 1, 6, 10, 0.5, 7, 2, ff=None), layer("attention", 8, 2, 9, 9, 0.3, 1, 0),
    layer("attention_2", 2, 1, 20, 12, 0.2, 1, 5), layer("attention", 3, 1, 16, 16, 0.3, 64, 64, ff=None),
    layer("attention", 2, 1, 300, 12, 0.05, 40, 3), layer("attention_2", 2, 1, 12, 300, 0.3, 40, 3), layer("attention", 2, 2, 30, 260, 0.2)])
def test_each_mechanism_alone(tmp_path, one):
    cfg = config([one], width=40, vocab=50)
    W = random_weights(cfg, 5)
    folder = write_folder(tmp_path / "m", cfg, W)
    tokens = ids(90, 50, 13)
    want, want16 = plain_logits(cfg, W, tokens), plain_logits(cfg, W, tokens, True)
    for dtype, w in (("float32", want), ("bfloat16", want16)):
        eng = engine(folder, dtype)
        assert rel(run(eng, [tokens]), w) < tol_of(dtype)
        assert rel(run(eng, [tokens[:30]] + [[t] for t in tokens[30:]]), w) < tol_of(dtype)


def test_values_are_mixed_with_the_first_mixing_layers_own(tmp_path):
    """Three layers of which the first does not mix: the second's values enter the third's, and the share decides how much;
    the second layer's own share enters nothing."""
    cfg = config([layer("attention", vdim=5), layer("attention_2", 2, 2, 8, 6, v_mix=True), layer("attention", 3, 1, 6, 12, v_mix=True)], 40, 50)
    tokens = ids(50, 50, 14)
    seen = []
    for name, first, later in (("a", 0.3, 0.5), ("b", -2.0, 0.5), ("c", 0.3, 0.0), ("d", 0.3, 1.0)):
        W = random_weights(cfg, 6)
        W["l1.mix.vmix"].fill_(first)
        W["l2.mix.vmix"].fill_(later)
        got = run(engine(write_folder(tmp_path / name, cfg, W)), cut(tokens, [20, 1, 1, 9]))
        assert rel(got, plain_logits(cfg, W, tokens)) < TOL_F32
        seen.append(got)
    assert rel(seen[1], seen[0]) < 1e-6 and rel(seen[2], seen[0]) > 1e-2 and rel(seen[3], seen[2]) > 1e-2


def test_a_share_beside_a_layer_that_does_not_mix_is_passed_over(tmp_path):
    cfg = config([layer("attention"), layer("attention_2")], 40, 50)
    W = random_weights(cfg, 6)
    tokens = ids(20, 50, 3)
    want = plain_logits(cfg, W, tokens)
    W["l0.mix.vmix"] = torch.tensor(0.5).to(torch.bfloat16)
    assert rel(run(engine(write_folder(tmp_path / "m", cfg, W)), [tokens]), want) < TOL_F32


# --------------------------------------------------------------------------- cutting, batches, slots and pages
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ALL))
def test_token_by_token_and_portions_equal_the_whole_prompt(folders, name, dtype):
    folder, cfg, W = folders[name]
    tokens = ids(161, cfg["vocab"], 15)
    want = plain_logits(cfg, W, tokens, dtype == "bfloat16")
    eng = engine(folder, dtype)
    for pieces in ([[t] for t in tokens], cut(tokens, [2] * 80), cut(tokens, [3, 61, 1, 64, 2]), cut(tokens, [130] + [1] * 30),
                   cut(tokens, [64, 64]), cut(tokens, [5] * 20)):
        assert rel(run(eng, pieces), want) < tol_of(dtype)
    assert all(g.pool.n_held == 0 for g in eng.cache.groups)


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "float32"), ("C", "bfloat16"), ("D", "bfloat16")])
def test_unequal_requests_in_a_batch_equal_each_alone_and_slots_are_used_again(folders, name, dtype):
    from scriptling_llm_lib_b200.engine.step import StepEntry
    folder, cfg, W = folders[name]
    reqs = [ids(n, cfg["vocab"], 20 + i) for i, n in enumerate((70, 3, 139, 1, 40, 200))]
    prompt = [60, 2, 100, 1, 33, 190]
    want = [plain_logits(cfg, W, r, dtype == "bfloat16") for r in reqs]
    eng = engine(folder, dtype, max_seqs=6, max_tokens=1024)
    for round_ in range(3):                     # the same slots and pages again, after other requests held them
        seqs = [eng.open() for _ in reqs]
        out = eng.step([StepEntry(s, r[:p], list(range(p))) for s, r, p in zip(seqs, reqs, prompt)]).cpu().double()
        got = [[o] for o in out.split(prompt)]
        pos = list(prompt)
        while True:
            for i, s in enumerate(seqs):
                if pos[i] == len(reqs[i]) and not s.closed:
                    s.close()
            live = [i for i in range(len(reqs)) if pos[i] < len(reqs[i])]
            if not live:
                break
            out = eng.step([StepEntry(seqs[i], [reqs[i][pos[i]]], [0]) for i in live]).cpu().double()
            for j, i in enumerate(live):
                got[i].append(out[j:j + 1])
                pos[i] += 1
        for i in range(len(reqs)):
            assert rel(torch.cat(got[i]), want[i]) < tol_of(dtype), (round_, i)
        reqs, prompt, want = reqs[::-1], prompt[::-1], want[::-1]
    assert eng.cache.slots.n_held == 0 and all(g.pool.n_held == 0 for g in eng.cache.groups)


@pytest.mark.parametrize("name,dtype", [("B", "float32"), ("C", "bfloat16")])
def test_a_step_may_mix_prompts_portions_and_single_tokens(folders, name, dtype):
    from scriptling_llm_lib_b200.engine.step import StepEntry
    folder, cfg, W = folders[name]
    a, b, c = (ids(n, cfg["vocab"], 70 + n) for n in (120, 45, 150))
    want = [plain_logits(cfg, W, r, dtype == "bfloat16") for r in (a, b, c)]
    eng = engine(folder, dtype)
    sa, sb, sc = eng.open(), eng.open(), eng.open()
    every = lambda s, t: StepEntry(s, t, list(range(len(t))))
    o1 = eng.step([every(sa, a[:90])]).cpu().double()
    o2 = eng.step([every(sb, b[:44]), every(sa, a[90:91]), every(sc, c[:70])]).cpu().double()
    o3 = eng.step([every(sc, c[70:150]), every(sb, b[44:]), every(sa, a[91:])]).cpu().double()
    assert rel(torch.cat([o1, o2[44:45], o3[81:]]), want[0]) < tol_of(dtype)
    assert rel(torch.cat([o2[:44], o3[80:81]]), want[1]) < tol_of(dtype)
    assert rel(torch.cat([o2[45:], o3[:80]]), want[2]) < tol_of(dtype)


def test_the_first_tokens_of_a_sequence(folders):
    for name in ("A", "B"):
        folder, cfg, W = folders[name]
        eng = engine(folder)
        for n in (1, 2, 3, 4, 5, 6):
            tokens = ids(n, cfg["vocab"], 30 + n)
            want = plain_logits(cfg, W, tokens)
            assert rel(run(eng, [tokens]), want) < TOL_F32
            assert rel(run(eng, [[t] for t in tokens]), want) < TOL_F32


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("C", "bfloat16"), ("D", "bfloat16")])
def test_long_decoding_gives_pages_back_and_keeps_the_first(folders, name, dtype):
    from scriptling_llm_lib_b200.engine.step import StepEntry
    folder, cfg, W = folders[name]
    tokens = ids(420, cfg["vocab"], 16)
    want = plain_logits(cfg, W, tokens, dtype == "bfloat16")
    eng = engine(folder, dtype, max_tokens=1024)
    seq = eng.open()
    got = [eng.step([StepEntry(seq, tokens[:5], list(range(5)))])]
    for t in tokens[5:]:
        got.append(eng.step([StepEntry(seq, [t], [0])]))
    assert rel(torch.cat(got).cpu().double(), want) < tol_of(dtype)
    for g in eng.cache.groups:
        held = [i for i, p in enumerate(g.pages[seq.slot]) if p >= 0]
        if g.need.kind == "full":
            assert held == list(range(7))
        else:
            first = max(0, len(tokens) - g.need.window + 1)
            assert held == [i for i in range(7) if 64 * i < g.need.keep or 64 * i + 63 >= first]
    assert any(len([p for p in g.pages[seq.slot] if p >= 0]) < 7 for g in eng.cache.groups)
    seq.close()


# --------------------------------------------------------------------------- a key that stands out
def loud_model(tmp_path, kind, dim, vdim, window, keep):
    """One attention layer whose queries all point along a head's first dim (their bias is large there) and whose keys have
    that dim from a channel only the last token id lights: whoever sees that token's key takes its values from it."""
    H, G, Wd = 4, 2, 64
    cfg = config([layer(kind, H, G, dim, vdim, 12.0 / dim, window, keep, False, None)], Wd, 40)
    W = random_weights(cfg, 7)
    c = Wd - 2                                       # the position vector hardly moves this channel
    W["embed"][:, c] = 0.0
    W["embed"][39, c] = 16.0
    for h in range(H):
        W["l0.mix.q"][h * dim:(h + 1) * dim] *= 0.1
        W["l0.mix.q.b"][h * dim] = 60.0
    for g in range(G):
        W["l0.mix.k"][g * dim] = 0.0
        W["l0.mix.k"][g * dim, c] = 12.0
        W["l0.mix.k.b"][g * dim] = 0.0
    return write_folder(tmp_path / "loud", cfg, W), cfg, W


@pytest.mark.parametrize("kind,dim,vdim,window,keep,dtype", [
    ("attention", 8, 12, 50, 3, "float32"), ("attention_2", 6, 5, 50, 3, "float32"), ("attention_2", 20, 20, 64, 65, "float32"),
    ("attention", 64, 64, 50, 3, "bfloat16"), ("attention_2", 128, 128, 130, 66, "bfloat16"), ("attention", 48, 32, 64, 64, "bfloat16"),
    ("attention_2", 96, 16, 65, 1, "bfloat16"), ("attention", 10, 6, 33, 5, "bfloat16")])
def test_one_loud_key_at_page_borders_and_at_every_edge(tmp_path, kind, dim, vdim, window, keep, dtype):
    folder, cfg, W = loud_model(tmp_path, kind, dim, vdim, window, keep)
    eng = engine(folder, dtype)
    n = 260
    base = ids(n, 39, 17)                            # never the loud token
    quiet = plain_logits(cfg, W, base)
    for p in sorted({0, keep - 1, keep, keep + 1, 63, 64, 65, 127, 128, 150} & set(range(n))):
        tokens = list(base)
        tokens[p] = 39
        want = plain_logits(cfg, W, tokens, dtype == "bfloat16")
        moved = (want - quiet).abs().amax(-1) / quiet.abs().amax(-1)
        edge = p + window                            # the first position that no longer sees it, unless it is kept
        assert float(moved[p + 1:min(edge, n)].median()) > 0.3
        if dtype == "float32" and edge < n:
            assert float(moved[edge - 1]) > 0.1
            assert (float(moved[edge:].min()) > 0.01) if p < keep else (float(moved[edge:].max()) < 1e-6)
        for pieces in ([tokens], [tokens[:p + 1]] + [[t] for t in tokens[p + 1:]], cut(tokens, [63, 2, 64, 41])):
            assert rel(run(eng, pieces), want) < tol_of(dtype), (p, len(pieces))


def attention_case(rng, L, H, G, hd, vd, dtype):
    """Queries, keys and values of one sequence, keys and values also on scattered pages whose unused rows are NaN."""
    q, k, v = (torch.from_numpy(rng.standard_normal(s)).to(dtype) for s in ((L, H, hd), (L, G, hd), (L, G, vd)))
    n_pages = (L + 63) // 64
    order = rng.permutation(n_pages + 3)[:n_pages]
    kp = torch.full((n_pages + 3, G, 64, hd), float("nan"), dtype=dtype)
    vp = torch.full((n_pages + 3, G, 64, vd), float("nan"), dtype=dtype)
    for j in range(L):
        kp[order[j // 64], :, j % 64], vp[order[j // 64], :, j % 64] = k[j], v[j]
    return q, k, v, kp.cuda(), vp.cuda(), [int(o) for o in order]


def attend_rows(q, k, v, rows, H, G, scale, window, keep, sink):
    """Formula for the given query rows, float64; `sink`: a logit per head or None."""
    out = torch.zeros((len(rows), H, v.shape[-1]), dtype=torch.float64)
    for a, i in enumerate(rows):
        js = [j for j in range(i + 1) if plain.sees(i, j, window, keep)]
        for h in range(H):
            s = (k[js, h // (H // G)].double() @ q[i, h].double()) * scale
            e = torch.exp(s - s.max())
            out[a, h] = (e / (e.sum() + (torch.exp(sink[h].double() - s.max()) if sink is not None else 0.0))) @ v[js, h // (H // G)].double()
    return out.reshape(len(rows), -1)


@pytest.mark.parametrize("H,G,hd,vd,window,keep,L,sinks,gated,dtype", [
    (4, 2, 64, 64, 100, 3, 400, True, True, "bfloat16"), (4, 4, 64, 64, 64, 64, 300, False, False, "bfloat16"),
    (6, 2, 128, 128, 40, 70, 390, True, True, "bfloat16"), (4, 2, 128, 128, 200, 1, 500, False, True, "bfloat16"),
    (3, 3, 128, 128, 33, 5, 385, True, False, "bfloat16"), (3, 1, 128, 128, 300, 129, 513, True, True, "bfloat16"),
    (6, 3, 88, 32, 120, 17, 420, True, True, "bfloat16"), (12, 1, 72, 24, 50, 140, 330, False, True, "bfloat16"),
    (2, 2, 256, 128, 64, 63, 260, True, False, "bfloat16"), (4, 1, 40, 104, 65, 65, 270, True, True, "bfloat16"),
    (4, 2, 8, 8, 20, 2, 150, True, True, "bfloat16"), (4, 2, 128, 64, None, 0, 300, True, True, "bfloat16"),
    (4, 2, 128, 128, None, 0, 300, False, True, "bfloat16"), (3, 1, 6, 10, 30, 4, 200, True, False, "bfloat16"),
    (4, 2, 12, 20, 50, 70, 300, True, False, "float32"), (5, 1, 128, 36, 65, 1, 260, False, False, "float32"),
    (3, 3, 7, 3, 64, 64, 200, True, False, "float32"), (2, 1, 256, 256, 90, 20, 210, True, False, "float32"),
    (2, 1, 512, 512, 40, 3, 130, True, False, "float32"), (2, 2, 16, 16, None, 0, 150, True, False, "float32")])
def test_attention_kernels_with_unequal_widths_a_window_and_kept_positions(H, G, hd, vd, window, keep, L, sinks, gated, dtype):
    """The part's own choice of kernel for a prompt, a portion of a few rows, a portion that lands on a cache, and a decode step,
    on scattered pages; keys at the window's edges and at the last kept positions are made to stand out."""
    from types import SimpleNamespace
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    from scriptling_llm_lib_b200.parts.attention import Attention
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    rng = np.random.default_rng(L + hd)
    q, k, v, kp, vp, order = attention_case(rng, L, H, G, hd, vd, dt)
    last = L - 1
    loud = [j for j in ((keep - 1, keep, last - window, last - window + 1) if window else (0, 63, 64)) if 0 <= j < last]
    for h in range(H):                                # the last query looks for these keys
        q[last, h] *= 0.2
        q[last, h, 0] = 6.0
    for n, j in enumerate(loud):
        k[j, :, 0] = 3.0 - 0.25 * n
        kp[order[j // 64], :, j % 64] = k[j].cuda()
    ks = KernelSet(dt)
    at = Attention(hidden=8, n_heads=H, n_kv_heads=G, head_dim=hd, v_dim=vd, position=None, q_name="q", k_name="k", v_name="v", o_name="o",
                   window=window, keep_first=keep, scale=0.7 / math.sqrt(hd) + 0.15, sink_value=0.0)
    at.sink = torch.from_numpy(rng.standard_normal(H)).float().cuda() if sinks else None
    err, tickets = torch.zeros(1, dtype=torch.int32, device="cuda"), torch.zeros(64, dtype=torch.int32, device="cuda")
    need = at.cache_need()
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    logits = torch.from_numpy(rng.standard_normal((L, H * vd + 8))).to(dt).cuda()

    def attend(first, n, decode):
        """Rows first .. first + n - 1 on what came before; pages no row of the step sees are marked as given back."""
        lo = first - window + 1 if window else 0
        table = [o if not window or 64 * i < keep or 64 * i + 63 >= lo else -1 for i, o in enumerate(order[:(first + n + 63) // 64])]
        ctx = SimpleNamespace(kernels=ks, is_decode=decode, n_seqs=1, max_new=n, seq_start=i32([0, n]), seq_pos0=i32([first]), err_flag=err,
                              pages_seen=lambda unit: min(len(table), need.pages_seen() or len(table)),
                              engine=SimpleNamespace(sm_count=148, tickets=lambda n: tickets))
        gate = logits[first:first + n, 8:] if gated else None
        return at._attend_general(q[first:first + n].reshape(n, -1).cuda(), gate, ctx, 0, kp, vp, i32([table])).double().cpu()

    def want(rows):
        w = attend_rows(q, k, v, rows, H, G, at.scale, window, keep, None if at.sink is None else at.sink.cpu())
        return w * torch.sigmoid(logits[rows, 8:].double().cpu()) if gated else w
    tol = 2e-5 if dtype == "float32" else 2.5e-2
    some = sorted({0, 1, 5, 63, 64, 65, L // 2, L - 66, L - 2, last} & set(range(L)))
    got = attend(0, L, False)
    assert int(err) == 0 and torch.isfinite(got).all()
    assert float((got[some] - want(some)).abs().max()) < tol
    for first, n in ((L - 3, 3), (L - 70, 70), (L - 9, 9)):
        rows = [r for r in (first, first + 1, last - 1, last)]
        assert float((attend(first, n, False)[[r - first for r in rows]] - want(rows)).abs().max()) < tol, (first, n)
    for r in (last, L // 2, 0, 1):
        assert float((attend(r, 1, True) - want([r])).abs().max()) < tol, r
    assert int(tickets.abs().sum()) == 0 and int(err) == 0


def test_decode_splits_of_any_number_give_the_same():
    """A window with kept pages over every number of splits, more than there are pages included; one sink however many."""
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    rng = np.random.default_rng(3)
    H, G, L, window, keep = 6, 2, 640, 200, 100
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")
    for hd, vd, dt in ((96, 40, torch.bfloat16), (128, 128, torch.bfloat16), (44, 28, torch.float32)):
        q, k, v, kp, vp, order = attention_case(rng, L, H, G, hd, vd, dt)
        sink = torch.full((H,), 1.5).cuda()
        want = attend_rows(q, k, v, [L - 1], H, G, 0.1, window, keep, sink.cpu())
        ks, out = KernelSet(dt), torch.empty(1, H * vd, dtype=dt, device="cuda")
        tickets = torch.zeros(8, dtype=torch.int32, device="cuda")
        for n_split in (1, 2, 3, 5, 6, 7, 13, 20):
            part = torch.full((H * n_split * (vd + 2),), float("nan"), device="cuda")
            args = (q[L - 1:].reshape(1, -1).cuda(), out, i32([L - 1]), i32([order]), kp, vp, part)
            if dt == torch.bfloat16:
                ks.decode.attn_decode_general(*args, tickets, 1, H, G, hd, vd, window, 0.1, n_split, keep=keep, sink=sink)
            else:
                ks.attn_decode_split(*args, 1, H, G, hd, window, 0.1, n_split, sink=sink, v_dim=vd, keep=keep)
            assert float((out.double().cpu() - want).abs().max()) < (2e-5 if dt == torch.float32 else 1e-2), (hd, n_split)


# --------------------------------------------------------------------------- the small kernels
@pytest.mark.parametrize("H,G,hd,vd,rot,interleaved", [(4, 2, 12, 8, 0, False), (3, 1, 7, 5, 0, False), (5, 5, 64, 16, 16, False),
                                                       (2, 1, 9, 3, 4, True), (6, 2, 128, 64, 128, True), (2, 2, 512, 260, 0, False),
                                                       (2, 1, 300, 8, 20, False), (20, 4, 128, 64, 0, False), (36, 9, 24, 40, 0, False),
                                                       (60, 4, 8, 8, 0, False)])
def test_the_store_kernel_adds_biases_norms_turns_mixes_and_fills_the_cache(H, G, hd, vd, rot, interleaved):
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    g = torch.Generator().manual_seed(H + hd)
    T, C = 5, (H + G) * hd + G * vd
    pos = [0, 3, 63, 64, 130]
    table = torch.tensor([[2, 0, 3]], dtype=torch.int32, device="cuda")
    ang = torch.rand((131, max(rot // 2, 1)), generator=g, dtype=torch.float64) * 6
    cs = torch.stack([torch.cos(ang), torch.sin(ang)], dim=-1).float().cuda()
    for dt, pad, tol in ((torch.float32, 4, 2e-6), (torch.bfloat16, 8, 1e-2), (torch.float32, 3, 2e-6)):
        k = KernelSet(dt).gate
        c = torch.randn((T, C + pad), generator=g).to(dt)
        bias = torch.randn(C, generator=g)
        for per_head in (True, False, None):
            for mode in (None, "keep", 0.3):
                widths = ((hd,) * 2 if per_head else (H * hd, G * hd)) if per_head is not None else ()
                qw, kw = (torch.rand(w, generator=g) + 0.5 for w in widths) if widths else (None, None)
                kept = torch.randn((T, G * vd), generator=g).to(dt)
                x = c[:, :C].double() + bias.double()
                q, kk, v = x[:, :H * hd], x[:, H * hd:(H + G) * hd], x[:, (H + G) * hd:]
                if widths:
                    q = plain.head_norms(q, qw.double(), H, 1e-3, not per_head)
                    kk = plain.head_norms(kk, kw.double(), G, 1e-3, not per_head)
                if rot:
                    def turn(y, n):
                        y = y.reshape(T, n, hd).clone()
                        a, b = (slice(0, rot, 2), slice(1, rot, 2)) if interleaved else (slice(0, rot // 2), slice(rot // 2, rot))
                        co, si = torch.cos(ang[pos])[:, None], torch.sin(ang[pos])[:, None]
                        u, w = y[..., a].clone(), y[..., b].clone()
                        y[..., a], y[..., b] = u * co - w * si, w * co + u * si
                        return y.reshape(T, -1)
                    q, kk = turn(q, H), turn(kk, G)
                stored = v if not isinstance(mode, float) else plain.mixed_values(v, kept.double(), mode)
                kp = torch.zeros((4, G, 64, hd), dtype=dt, device="cuda")
                vp = torch.zeros((4, G, 64, vd), dtype=dt, device="cuda")
                q_out, kd = torch.empty((T, H * hd), dtype=dt, device="cuda"), kept.cuda()
                dev = lambda t: t.cuda() if t is not None else None
                k.qk_norm_store(c.cuda()[:, :C], q_out, torch.tensor(pos, dtype=torch.int32).cuda(), torch.zeros(T, dtype=torch.int32).cuda(), table,
                                cs if rot else None, kp, vp, H, G, hd, vd, rot, interleaved, dev(qw), dev(kw), 1e-3, bias=bias.cuda(),
                                per_head=bool(per_head), value_mix=None if mode is None else (kd, None if mode == "keep" else mode))
                near = lambda got, want: float((got.double().cpu() - want).abs().max()) < tol * max(1.0, float(want.abs().max()))
                assert near(q_out, q)
                for t, p in enumerate(pos):
                    page = int(table[0, p // 64])
                    assert near(kp[page, :, p % 64].reshape(-1), kk[t]) and near(vp[page, :, p % 64].reshape(-1), stored[t])
                if mode == "keep":
                    assert near(kd, v)
                assert int((kp != 0).any(-1).sum()) == T * G


@pytest.mark.parametrize("d,P", [(128, 1), (2048, 3), (35, 2), (1030, 1), (4096, 2)])
def test_the_sum_of_a_normed_addend_with_a_bias_and_the_copy(d, P):
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    g = torch.Generator().manual_seed(d)
    T = 7
    for dt in (torch.float32, torch.bfloat16):
        k = KernelSet(dt).gate
        x, y = torch.randn((T, d), generator=g), torch.randn((P, T, d), generator=g) if P > 1 else torch.randn((T, d), generator=g).to(dt)
        b, w, w2 = (torch.randn(d, generator=g) for _ in range(3))
        s = (y.double().sum(0) if P > 1 else y.double()) + b.double()
        want = x.double() + plain.rms_div(s, 1e-5) * w.double()
        for how in ("alone", "copy", "norm", "rows"):
            xd = x.cuda()
            rows = torch.tensor([6, 2], dtype=torch.int32).cuda() if how == "rows" else None
            out = torch.empty((2 if how == "rows" else T, d), dtype=dt, device="cuda")
            kw = {"copy": dict(copy=out), "norm": dict(norm=(w2.cuda(), 1e-5, out)), "rows": dict(norm=(w2.cuda(), 1e-5, out), rows=rows)}.get(how, {})
            k.add_rms_normed(xd, y.cuda(), w.cuda(), 1e-5, y_bias=b.cuda(), **kw)
            unit = 1e-5 if dt == torch.float32 else 2.0 ** -8       # of an element: bfloat16 keeps eight bits
            if how != "rows":
                assert float((xd.double().cpu() - want).abs().max()) < 1e-5
            if how == "copy":
                assert torch.equal(out, xd.to(dt))
            elif how != "alone":
                n = plain.rms_div(want, 1e-5) * w2.double()
                n = n[[6, 2]] if how == "rows" else n
                assert bool(((out.double().cpu() - n).abs() <= unit * n.abs() + 1e-5).all())


def test_the_embedding_with_positions_far_out():
    from types import SimpleNamespace
    from scriptling_llm_lib_b200.csrc.bindings import KernelSet
    from scriptling_llm_lib_b200.parts.embedding import SinusoidEmbedding
    g = torch.Generator().manual_seed(1)
    err = torch.zeros(1, dtype=torch.int32, device="cuda")
    pos = [0, 1, 2, 63, 64, 65, 1000, 4095, 131071]
    for width in (9, 64, 250):
        for dt in (torch.float32, torch.bfloat16):
            e = SinusoidEmbedding(30, width, "e")
            table = torch.randn((30, width), generator=g).to(dt)
            e.bind({"e": table.cuda()}, dt, "cuda")
            e.prepare(131072, "cuda")
            tok = [(7 * p + 3) % 30 for p in pos]
            ks = KernelSet(dt)
            ctx = SimpleNamespace(kernels=ks, dtype=dt, err_flag=err, tok_pos=torch.tensor(pos, dtype=torch.int32).cuda())
            x = e.forward(torch.tensor(tok, dtype=torch.int32).cuda(), ctx).double().cpu()
            want = torch.stack([table[t].double() + plain.sinusoid(p, width) for t, p in zip(tok, pos)])
            assert float((x - want).abs().max()) < 1e-6 and int(err) == 0


# --------------------------------------------------------------------------- the entry point
def test_greedy_generation_through_the_entry_point(folders):
    from scriptling_llm_lib_b200 import llm
    folder, cfg, W = folders["A"]
    prompt = ids(41, cfg["vocab"], 19)
    for dtype in ("float32", "bfloat16"):
        out = llm.generate(str(folder), prompt, max_tokens=30, strategy="greedy", dtype=dtype)
        tokens = list(prompt)
        for t in out:
            lg = plain_logits(cfg, W, tokens)[-1]
            top2 = lg.topk(2).values
            if dtype == "float32" or float(top2[0] - top2[1]) > 0.1 * float(lg.abs().max()):
                assert int(lg.argmax()) == t
            tokens.append(t)
        assert len(out) == 30
        llm.unload()


def test_a_batch_of_unequal_prompts_generates_what_each_alone_does(folders):
    from scriptling_llm_lib_b200 import llm
    folder, cfg, W = folders["B"]
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
    cfg_path.write_text(json.dumps(CFG_C))
    got = run(engine(f"random:{cfg_path}:3", "bfloat16"), [ids(40, CFG_C["vocab"], 1)])
    assert torch.isfinite(got).all() and float(got.abs().max()) > 0
    root = Path(__file__).resolve().parent.parent
    r = subprocess.run([sys.executable, "-m", "scriptling_llm_lib_b200", "-model", f"random:{cfg_path}:3", "-prompt", "1,2,3",
                        "-tokens", "4"], cwd=root, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr


def test_trace_replay_writes_the_logits_of_the_wanted_places(folders, tmp_path):
    import subprocess
    import sys
    from pathlib import Path
    folder, cfg, W = folders["B"]
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
    read = lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V).copy()).double()
    assert rel(read(0), wa[[0, 24]]) < TOL_F32
    assert rel(read(1), torch.stack([wa[25], wb[8]])) < TOL_F32
    assert not (out / "2.f32").exists()
    assert rel(read(3), wa[29:30]) < TOL_F32

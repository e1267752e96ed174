"""Token embedding and output head.

x[i, :] = E[id_i, :] (model_f32.go:363-369), which a model may scale; logits = n W^T with W the embedding when
the head is tied (model_f32.go:147-162, :519-524). The reference skips ids outside the table and
leaves stale data in the row; here such an id is an error before anything runs. Both are parts
like the others, named in a layout by kind ("token_embedding", "linear_head"): a model that scales
its embedding or caps its logits registers parts of its own.
"""
from __future__ import annotations

import torch

from ..weights.spec import TensorSpec
from .base import EMBEDDINGS, HEADS, Embedding, Head, PartSpec
from .linear import Linear


EMBEDDING_OUTPUT = "embedding_output"     # the key of the step's embedding output among what its parts share


class TokenEmbedding(Embedding):
    """x = scale * E[token]. With `keep_output` the step keeps a copy of x for a part that adds it to the stream again
    between two layers (`embedding_again`); the kernel writes both. Scale and copy are absent in the reference."""

    def __init__(self, vocab: int, width: int, name: str, scale: float = 1.0, keep_output: bool = False):
        self.vocab, self.width, self.name = vocab, width, name
        self.scale, self.keep_output = float(scale), bool(keep_output)
        self.table = None

    def _copy(self, out, ctx):
        """Where the kernel puts the copy of its rows that the step keeps (None: nobody asks for one)."""
        if not self.keep_output:
            return None
        ctx.scratch[EMBEDDING_OUTPUT] = torch.empty_like(out)
        return ctx.scratch[EMBEDDING_OUTPUT]

    def tensor_specs(self):
        return [TensorSpec(self.name, (self.vocab, self.width))]

    def elements_read_per_step(self) -> int:
        return 0                                    # a step reads one row per token, not the table

    def bind(self, tensors, dtype, device):
        self.table = tensors[self.name]

    def forward(self, ids, ctx):
        out = torch.empty((ids.shape[0], self.width), dtype=torch.float32, device=ids.device)
        k = ctx.kernels if self.table.dtype == ctx.dtype else ctx.kernels_f32
        k.embed_rows(ids, self.table, out, ctx.err_flag, scale=self.scale, copy=self._copy(out, ctx))
        return out


class SinusoidEmbedding(TokenEmbedding):
    """x = E[token] + s(p): at position p of its sequence a token takes a fixed vector (absent in the reference),
    s_2i = sin(p / base^(2i / width)) and s_2i+1 = cos of the same angle. Angles are made on the host in float64, as
    (sin, cos) of the positions 0, 64, 128, ... and of 0 .. 63; the kernel puts position 64 a + b together from the two."""
    STRIDE = 64

    def __init__(self, vocab: int, width: int, name: str, base: float = 10000.0):
        super().__init__(vocab, width, name)
        self.base = float(base)
        self.coarse = self.fine = None

    def prepare(self, max_positions, device):
        pairs = (self.width + 1) // 2
        freq = torch.pow(torch.tensor(self.base, dtype=torch.float64), -2.0 * torch.arange(pairs, dtype=torch.float64) / self.width)

        def table(positions):
            angle = positions.to(torch.float64)[:, None] * freq[None, :]
            return torch.stack([torch.sin(angle), torch.cos(angle)], dim=-1).to(torch.float32).to(device).contiguous()
        self.coarse = table(torch.arange(-(-max_positions // self.STRIDE)) * self.STRIDE)
        self.fine = table(torch.arange(self.STRIDE))

    def forward(self, ids, ctx):
        out = torch.empty((ids.shape[0], self.width), dtype=torch.float32, device=ids.device)
        k = ctx.kernels if self.table.dtype == ctx.dtype else ctx.kernels_f32
        k.embed_rows_sinusoid(ids, ctx.tok_pos, self.table, self.coarse, self.fine, out, ctx.err_flag)
        return out


class PairHashEmbedding(TokenEmbedding):
    """x = scale * E[token] + P[r]: a second table P [buckets + 1, width] is looked up by the pair (previous token, token),
    r = (previous * mul_prev + token * mul_cur) mod buckets, and by its last row, r = buckets, for a sequence's first token
    (absent in the reference). The previous token of a step's first row is per-sequence state: one int32 per slot
    (`state_need`), read and then set to the run's last token by the embedding kernel itself, so prompts in portions,
    decode steps and replayed steps all find it on the device."""

    def __init__(self, vocab: int, width: int, name: str, pair_name: str, buckets: int, mul_prev: int, mul_cur: int,
                 scale: float = 1.0, keep_output: bool = False):
        super().__init__(vocab, width, name, scale, keep_output)
        if buckets < 1 or mul_prev < 0 or mul_cur < 0:
            raise ValueError(f"a pair table of {buckets} buckets with multipliers {mul_prev}, {mul_cur}")
        self.pair_name = pair_name
        self.buckets, self.mul_prev, self.mul_cur = int(buckets), int(mul_prev), int(mul_cur)
        self.pair_table = None

    def tensor_specs(self):
        return [TensorSpec(self.name, (self.vocab, self.width)), TensorSpec(self.pair_name, (self.buckets + 1, self.width))]

    def state_need(self):
        from ..cache.needs import StateNeed
        return StateNeed((), torch.int32)

    def bind(self, tensors, dtype, device):
        self.table, self.pair_table = tensors[self.name], tensors[self.pair_name]
        if self.table.dtype != self.pair_table.dtype:
            raise ValueError(f"{self.name} and {self.pair_name} are stored in different precisions")

    def forward(self, ids, ctx):
        out = torch.empty((ids.shape[0], self.width), dtype=torch.float32, device=ids.device)
        k = ctx.kernels if self.table.dtype == ctx.dtype else ctx.kernels_f32
        k.embed_pair_rows(ids, ctx, self.table, self.pair_table, self.buckets, self.mul_prev, self.mul_cur,
                          ctx.unit_state(EMBEDDING_STATE), out, ctx.err_flag, scale=self.scale, copy=self._copy(out, ctx))
        return out


EMBEDDING_STATE = "embedding"      # the key of the embedding's per-sequence state among the cache units' states


class OutputHead(Head):
    """Logits in float32 for the rows it is given. `tied`: the matrix is another part's tensor (the
    embedding's), named by `weight_name`, and is not asked of the weight file a second time. `softcap` (absent in the
    reference): the logits leave as cap * tanh(logits / cap). `scale` (absent in the reference): the logits are multiplied by
    it (before a cap)."""

    def __init__(self, vocab: int, width: int, weight_name: str, tied: bool = False, softcap: float | None = None,
                 scale: float | None = None):
        self.vocab, self.width, self.tied = vocab, width, tied
        self.scale = float(scale) if scale is not None else 1.0
        self.softcap = float(softcap) if softcap else None
        if self.softcap is not None and not self.softcap > 0:
            raise ValueError(f"a cap on the logits must be positive, got {softcap}")
        self.linear = Linear([weight_name], [vocab], width)

    def tensor_specs(self):
        return [] if self.tied else self.linear.tensor_specs()

    def elements_read_per_step(self) -> int:
        return self.vocab * self.width

    def bind(self, tensors, dtype, device):
        self.linear.bind(tensors, dtype, device)

    def forward(self, normed, ctx):
        logits = self.linear.forward(normed, ctx, out_dtype=torch.float32)
        if self.softcap is not None or self.scale != 1.0:
            ctx.kernels.gate.softcap(logits, self.softcap, self.scale)
        return logits


EMBEDDINGS.register("token_embedding", TokenEmbedding)
EMBEDDINGS.register("sinusoid_embedding", SinusoidEmbedding)
EMBEDDINGS.register("pair_hash_embedding", PairHashEmbedding)
HEADS.register("linear_head", OutputHead)


def token_embedding(vocab: int, width: int, name: str, scale: float = 1.0, keep_output: bool = False) -> PartSpec:
    params = dict(vocab=vocab, width=width, name=name)
    if scale != 1.0:
        params["scale"] = scale
    if keep_output:
        params["keep_output"] = True
    return PartSpec("token_embedding", params)


def linear_head(vocab: int, width: int, weight_name: str, tied: bool = False, softcap: float | None = None,
                scale: float | None = None) -> PartSpec:
    params = dict(vocab=vocab, width=width, weight_name=weight_name, tied=tied)
    if softcap:
        params["softcap"] = softcap
    if scale is not None and scale != 1.0:
        params["scale"] = scale
    return PartSpec("linear_head", params)

"""The state-space recurrence with one decay per head and token (the mixer of Mamba-2).

The input projection Win h is [z: inner | x: inner | B: G N | C: G N | dt: heads], inner = heads * head_dim. On x, B and C
together runs a short causal convolution over time, one filter and one bias per channel, followed by SiLU. Per head i, whose
group is i // (heads / G): dt = softplus(dt + dt_bias), and the state S [N, head_dim] follows
S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x. The heads' y side by side, times silu(z), pass an RMS norm taken
apart in `norm_groups` equal runs of columns (one weight per column), and Wo maps them back.

State per sequence: S [heads, N, head_dim] in float32 (zero at the start) and the convolution's last taps - 1 inputs. The
projections and the convolution with its SiLU run in the engine's dtype; step sizes, decays, exponentials, state and
read-out are float32 (csrc/ssd_kernels.cuh). A decode step or a short run walks token by token; a long run in bfloat16 goes
through the tensor cores in chunks. Where the norm is over the whole row and the output product can take over its second
half (base.py: Folded), the recurrence's kernel writes y silu(z) times the norm's weight and the sums of squares, and the
norm needs no kernel. Not in the reference.
"""
from __future__ import annotations

import torch

from ..cache.needs import StateNeed
from ..weights.spec import TensorSpec
from .base import MIXERS, Folded, Mixer
from .conv import CausalConv
from .linear import Linear


class Mamba2(Mixer):
    graph_safe = True
    MAX_STATE = 1024

    def __init__(self, hidden: int, n_heads: int, head_dim: int, n_state: int, n_groups: int, conv_taps: int, norm_groups: int,
                 norm_eps: float, in_name: str, conv_name: str, conv_bias_name: str, dt_bias_name: str, a_log_name: str, d_name: str,
                 norm_name: str, o_name: str):
        if not 1 <= n_state <= self.MAX_STATE:
            raise ValueError(f"a state of {n_state}: the recurrence's kernels take 1..{self.MAX_STATE}")
        if n_heads % n_groups:
            raise ValueError(f"{n_heads} heads do not fall into {n_groups} equal groups")
        self.H, self.V, self.N, self.G = n_heads, head_dim, n_state, n_groups
        self.inner = n_heads * head_dim
        if self.inner % norm_groups:
            raise ValueError(f"{self.inner} columns do not fall into {norm_groups} equal runs")
        self.norm_groups, self.eps = int(norm_groups), float(norm_eps)
        self.conv_width = self.inner + 2 * n_groups * n_state
        self.in_proj = Linear([in_name], [self.inner + self.conv_width + n_heads], hidden)
        self.conv = CausalConv([conv_name], [self.conv_width], conv_taps, bias_name=conv_bias_name, act="silu")
        self.out = Linear([o_name], [hidden], self.inner)
        self.names = dict(dt_bias=dt_bias_name, a_log=a_log_name, d=d_name, norm=norm_name)

    def tensor_specs(self):
        n = self.names
        return self.in_proj.tensor_specs() + self.conv.tensor_specs() + [
            TensorSpec(n["dt_bias"], (self.H,), init="bias"), TensorSpec(n["a_log"], (self.H,), init="log_rate"),
            TensorSpec(n["d"], (self.H,), init="norm_weight"), TensorSpec(n["norm"], (self.inner,), init="norm_weight"),
        ] + self.out.tensor_specs()

    def bind(self, tensors, dtype, device):
        for part in (self.in_proj, self.conv, self.out):
            part.bind(tensors, dtype, device)
        w = self.in_proj.weight
        if w.shape[0] % 8:      # rows of zeros up to a multiple of 8, so that the product's rows stay aligned
            self.in_proj.weight = torch.cat([w, w.new_zeros((-w.shape[0] % 8, w.shape[1]))]).contiguous()
        self.dt_bias, self.a_log, self.d, self.norm_w = (tensors[self.names[k]].float().contiguous()
                                                         for k in ("dt_bias", "a_log", "d", "norm"))

    def state_need(self):
        need = {"S": StateNeed((self.H, self.N, self.V), torch.float32)}
        conv = self.conv.state_need()
        if conv is not None:
            need["conv"] = conv
        return need

    def forward(self, x, ctx, unit, writes, state=None):
        st = state if state is not None else ctx.unit_state(unit)
        T, I = x.shape[0], self.inner
        proj = self.in_proj.forward(x, ctx)                                      # [T, z | x B C | dt], raw
        xbc = self.conv.forward(proj[:, I:I + self.conv_width], st.get("conv"), ctx, x.dtype)
        at = I + self.conv_width
        k = ctx.kernels.ssd
        y = torch.empty((T, I), dtype=x.dtype, device=x.device)
        fold = self.norm_groups == 1 and not ctx.is_decode and self.out.fold_path(ctx, T, ctx.dtype) is not None
        sumsq = k.scan(xbc, proj[:, at:at + self.H], self.dt_bias, self.a_log, self.d, proj[:, :I], st["S"], ctx, y, self.H, self.G,
                       self.V, self.N, weight=self.norm_w if fold else None)
        if fold:
            return self.out.forward_folded(Folded(y, sumsq, I, self.eps), ctx)
        k.group_norm(y, self.norm_w, y, self.norm_groups, self.eps)
        return self.out.forward(y, ctx, partials_ok=True)


MIXERS.register("mamba2", Mamba2)

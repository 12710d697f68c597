"""A selective state-space mixer with one scalar decay per head and token (state-space duality, "Mamba-2").

h -> one stacked product gives z (heads x value_dim), x (heads x value_dim), B and C (groups x state_dim each) and one step
logit per head, as float32 sums. x, B and C pass one causal convolution per channel (with bias; its last inputs live in the
request's state slot) and SiLU. Per head, with S [state_dim, value_dim] from the slot, token by token:

    dt = softplus(dt_logit + dt_bias)
    S <- exp(-exp(A_log) dt) S + dt B x^T                        (heads share B and C in groups)
    y = S^T C + D x

-> u = y * silu(z) over the concatenated heads, RMS-normed in `norm_groups` equal parts (each by its own root mean square),
times a gain per channel, projected by W_o. The state, step sizes, decays, the read-out, the gate and the norm are float32
whatever the activation dtype. Single tokens run one kernel from the projection's row to y; prompt portions in bfloat16 run
chunks of tokens side by side on the tensor cores; float32 portions (and sizes the chunks do not take) walk token by token.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..weights.binding import ParamSpec
from .base import Mixer, StateSpec, register_part
from .linear import linear


class StateSpace(Mixer):
    accepts_deferred_input = True
    launches_through_kernels_only = True
    can_overwrite_output = True
    can_take_projected_input = True

    def __init__(self, spec, *, hidden_size: int):
        super().__init__(spec)
        s = spec
        if s.num_heads <= 0 or s.num_groups <= 0 or s.num_heads % s.num_groups:
            raise ValueError(f"num_heads {s.num_heads} is not a multiple of num_groups {s.num_groups}")
        if not 0 < s.state_dim <= 1024 or s.value_dim <= 0:
            raise ValueError(f"state_dim {s.state_dim} must lie in 1..1024 and value_dim {s.value_dim} be positive")
        if not 1 <= s.conv_taps <= 64:
            raise ValueError(f"conv_taps {s.conv_taps} must lie in 1..64")
        self.hidden_size = hidden_size
        self.H, self.G, self.N, self.V, self.taps = s.num_heads, s.num_groups, s.state_dim, s.value_dim, s.conv_taps
        self.inner = self.H * self.V
        if s.norm_groups <= 0 or self.inner % s.norm_groups:
            raise ValueError(f"{self.inner} channels do not form {s.norm_groups} equal parts")
        # columns of the stacked product: z | x | B | C | step logits
        self.conv_cols = self.inner + 2 * self.G * self.N
        self.dt_at = self.inner + self.conv_cols
        self.in_cols = self.dt_at + self.H
        self.conv_state_at = -(-self.H * self.N * self.V // 4) * 4       # (16-byte rows, as the state's own)

    def input_pieces(self):
        return (self.in_cols,)

    def param_specs(self):
        d = self.hidden_size
        specs = {
            "conv": ParamSpec((self.conv_cols, self.taps), role="gain", init=(0.0, 0.5)),
            "conv_bias": ParamSpec((self.conv_cols,), role="gain", init=(0.0, 0.2)),
            "dt_bias": ParamSpec((self.H,), role="gain", init=(-2.0, 1.0)),
            "a_log": ParamSpec((self.H,), role="gain", init=(0.0, 1.0)),
            "skip": ParamSpec((self.H,), role="gain", init=(1.0, 0.3)),
            "out_norm": ParamSpec((self.inner,), role="gain"),
            "wo": ParamSpec((d, self.inner)),
        }
        if not self.projected_input:
            specs["w_in"] = ParamSpec((self.in_cols, d))
        return specs

    def cache_spec(self):
        """One float32 row per request: S [heads, state_dim, value_dim], then the convolution's last inputs in a ring of
        `taps` rows [taps, x | B | C channels]."""
        return StateSpec((-(-(self.conv_state_at + self.taps * self.conv_cols) // 4) * 4,), torch.float32)

    def forward(self, ctx, h, residual, cache, writes_cache: bool) -> None:
        n = h.shape[0]
        p, f32 = self.params, torch.float32
        if self.projected_input:
            proj = h
        else:
            ld = -(-self.in_cols // 4) * 4                  # rows of the float32 buffer start 16-byte aligned
            proj = ctx.scratch("ssd_proj", (n, ld), f32)[:, :self.in_cols]
            linear(ctx, h, p["w_in"], proj)
        xbc, dt = proj[:, self.inner:self.dt_at], proj[:, self.dt_at:]
        y = ctx.scratch("ssd_y", (n, self.inner), f32)
        self.recur(ctx, xbc, dt, y, cache.state, writes_cache)
        att = ctx.scratch("att", (n, self.inner))
        kernels.gate_group_norm(y, proj[:, :self.inner], p["out_norm"], att, self.spec.norm_groups, self.spec.norm_eps, ctx.positions)
        linear(ctx, att, p["wo"], residual, accumulate=not getattr(ctx, "overwrite_output", False))

    def recur(self, ctx, xbc, dt, y, state, writes_cache: bool) -> None:
        """y from the projection's columns x | B | C and the step logits. In a mixed batch the single-token requests at its
        head take the decoding kernel, the portions behind them the other form."""
        n, p = xbc.shape[0], self.params
        k = ctx.seq_start_pos.shape[0] if ctx.decode_only else ctx.leading_single
        if k:
            kernels.ssd_decode(xbc, dt, p["conv"], p["conv_bias"], p["dt_bias"], p["a_log"], p["skip"], state, self.conv_state_at, y,
                               ctx.seq_first_row[:k + 1], ctx.seq_start_pos[:k], ctx.seq_slots[:k], self.H, self.G, self.N, self.V,
                               writes_cache, ctx.status)
        if ctx.decode_only or k >= ctx.seq_start_pos.shape[0]:
            return
        chunked = kernels.ssd_chunks_supported(ctx.dtype, self.N, self.V)
        ld = -(-self.conv_cols // 8) * 8
        act = ctx.scratch("ssd_xbc", (n, ld), ctx.dtype if chunked else torch.float32)[:, :self.conv_cols]
        kernels.ring_conv(xbc, p["conv"], p["conv_bias"], act, state, self.conv_state_at, ctx.row_seq, ctx.positions, ctx.seq_first_row,
                          ctx.seq_start_pos, ctx.seq_slots, writes_cache, ctx.status, first_row=k, first_seq=k)
        args = (act, dt, p["dt_bias"], p["a_log"], p["skip"], state, y, ctx.seq_first_row[k:], ctx.seq_start_pos[k:], ctx.seq_slots[k:])
        if not chunked:
            kernels.ssd_walk(*args, self.H, self.G, self.N, self.V, writes_cache, ctx.status)
            return
        chunks = kernels.ssd_chunks_needed(n, ctx.seq_start_pos.shape[0] - k)
        own = ctx.scratch("ssd_chunk_state", (chunks, self.H * self.N * self.V), torch.float32, grow=True)
        steps = ctx.scratch("ssd_chunk_steps", (chunks, self.H * 2 * kernels.ssd_chunk_rows()), torch.float32, grow=True)
        kernels.ssd_chunks(*args, ctx.max_rows_per_seq, self.H, self.G, self.N, self.V, writes_cache, ctx.status, own, steps)


register_part("mixer", "state_space", StateSpace, replace=True)

"""The state-space mixer with one scalar decay per head (the Mamba-2 kind).

With mixer input h, H heads of P channels (C = H P in all), N states per channel, and G groups of heads that share their maps:
    [z | x | B | C | dt] = W_in h                                C, C, G N, G N and H entries
    x, B, C  = silu(causal_conv([x | B | C]) + b)                per channel over the request's tokens
    dt       = softplus(dt + dt_bias)                            one step size per head
    S       <- exp(-exp(A_log) dt) S + dt B x^T ,   y = S^T C + D x      per head, S [N, P]
    out      = W_o ( rms_norm(y * silu(z), in norm_groups equal parts) * w )
A request's state is S in 32 bit (a channel's N entries side by side) and the convolution's last inputs, both zero at its start, one
pair per run of the layer; a step continues from what the request's earlier steps left, so a prompt may be cut anywhere.

W_in's rows are put into the order x | B | C | z | dt when they are bound, so that the convolution's inputs come first.  Step sizes,
decays, the recurrence and the norm are 32 bit whatever the compute type (``csrc/state_space.cu``): steps of single tokens and short
portions take the tokens in turn with the state in registers, long portions run in chunks of 32 tokens.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from . import linear
from .base import MIXERS, Mixer, StateSpec, TensorSpec
from .chunks import chunk_layout

PARALLEL_FROM = 33      # portions of at least this many tokens run in chunks
CONV_STATE = "conv"
STATE = "ssd"


@MIXERS.register("state_space")
class StateSpace(Mixer):
    """Tensor names under ``prefix``: ``in`` [2 C + 2 G N + H, d], ``conv`` [C + 2 G N, taps], ``conv.b`` [C + 2 G N], ``dt_bias``, ``A_log``,
    ``D`` [H], ``norm`` [C], ``o`` [d, C]."""

    def __init__(self, prefix: str, width: int, heads: int, head_dim: int, state: int, groups: int, conv: int, norm_groups: int, eps: float):
        self.prefix, self.width = prefix, int(width)
        self.heads, self.P, self.N, self.groups, self.taps = int(heads), int(head_dim), int(state), int(groups), int(conv)
        self.norm_groups, self.eps = int(norm_groups), float(eps)
        self.inner = self.heads * self.P
        self.channels = self.inner + 2 * self.groups * self.N
        if self.heads % self.groups:
            raise ValueError(f"{heads} heads are no multiple of {groups} groups")
        if self.inner % self.norm_groups:
            raise ValueError(f"{self.inner} channels do not split into {norm_groups} equal parts")
        if self.taps < 1:
            raise ValueError("the convolution needs at least one tap")
        self.w_in = self.w_o = self.conv_w = self.conv_b = self.dt_bias = self.A_log = self.D = self.norm_w = None

    def tensor_specs(self):
        p, d, C, ch, H = self.prefix, self.width, self.inner, self.channels, self.heads
        return [TensorSpec(p + "in", (C + ch + H, d)), TensorSpec(p + "conv", (ch, self.taps), kind="vector", init="uniform:-0.5:0.5"),
                TensorSpec(p + "conv.b", (ch,), kind="vector", init="uniform:-0.1:0.1"),
                TensorSpec(p + "dt_bias", (H,), kind="vector", init="uniform:-5:-1"),
                TensorSpec(p + "A_log", (H,), kind="vector", init="uniform:0:2"), TensorSpec(p + "D", (H,), kind="vector", init="norm"),
                TensorSpec(p + "norm", (C,), kind="vector", init="norm"), TensorSpec(p + "o", (d, C))]

    def bind(self, tensors):
        p, C, ch = self.prefix, self.inner, self.channels
        f = lambda n: tensors[p + n].float().contiguous()   # noqa: E731  (what the recurrence reads is kept in 32 bit)
        w = tensors[p + "in"]
        self.w_in = linear.padded_rows(torch.cat([w[C:C + ch], w[:C], w[C + ch:]], dim=0))
        self.w_o = tensors[p + "o"]
        self.conv_w, self.conv_b, self.dt_bias, self.A_log, self.D, self.norm_w = (f("conv"), f("conv.b"), f("dt_bias"), f("A_log"), f("D"), f("norm"))

    def run_state_specs(self):
        return {CONV_STATE: StateSpec((max(self.taps - 1, 1), self.channels), torch.float32, 0.0),
                STATE: StateSpec((self.heads, self.P, self.N), torch.float32, 0.0)}

    def forward(self, ctx, x, cache):
        H, G, N, P, C = self.heads, self.groups, self.N, self.P, self.inner
        T = x.shape[0]
        st = cache.state
        rows = dict(row_slot=ctx.row_slot, row_q_start=ctx.row_q_start, row_q_len=ctx.row_q_len)
        src = linear.linear(ctx, x, self.w_in)                                  # [T, channels + C + H]: x | B | C | z | dt
        at = lambda column: src.data_ptr() + column * src.element_size()       # noqa: E731
        xbc = torch.empty((T, self.channels), dtype=x.dtype, device=x.device)
        ops.conv_silu(src, src.shape[1], self.conv_w, self.conv_b, st[CONV_STATE], xbc, tok_row=ctx.tok_row, single=ctx.decode_only, **rows)
        y = torch.empty((T, C), dtype=torch.float32, device=x.device)
        args = (xbc, at(self.channels + C), src.shape[1], self.A_log, self.dt_bias, self.D, st[STATE], y)
        sizes = dict(H=H, G=G, N=N, P=P)
        if not ctx.replayable and ctx.max_q_len >= PARALLEL_FROM and ops.state_space_chunked_supported(N, P, x.dtype):
            base, total, most = chunk_layout(ctx, ops.state_space_chunk())
            per = ops.state_space_chunk_floats(H, G)
            bound = (-(-ctx.max_step_tokens // ops.state_space_chunk()) + ctx.max_rows) * per
            work = ctx.scratch("state_space.chunks", (total * per,), torch.float32, bound=(bound,))
            ops.state_space_chunked(*args, work, base, total, most, **sizes, **rows)
        else:
            if ctx.decode_only:
                rows["row_q_len"] = None
            ops.state_space(*args, **sizes, **rows)
        gated = torch.empty((T, C), dtype=x.dtype, device=x.device)
        ops.gated_rms_norm(y, at(self.channels), src.shape[1], self.norm_w, gated, self.eps, group=C // self.norm_groups, gate_first=True)
        return linear.linear(ctx, gated, self.w_o)

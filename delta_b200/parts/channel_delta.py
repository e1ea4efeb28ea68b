"""The gated delta rule with one decay per head and key channel ("Kimi delta attention" is of this kind).

With mixer input h, H heads on ``kv_heads`` query/key heads (head i reads query/key head i // (H / kv_heads)), key size dk and
value size dv:
    q, k, v = silu(conv(W_q h)), silu(conv(W_k h)), silu(conv(W_v h))        a short causal convolution per channel
    q, k    = x / sqrt(sum(x^2) + guard) per head,   q also times dk^(-1/2)
    beta    = sigmoid(W_b h)                                                  one per head
    g       = exp(-exp(A_log) * softplus(W_a2 W_a1 h + dt_bias))              one per head and key channel
    S <- diag(g) S ;   u = beta (v - S^T k) ;   S <- S + k u^T ;   o = S^T q  per head, token by token
    out     = W_o ( o / rms(o per head) * w * sigmoid(W_g2 W_g1 h) )
A request's state is S in 32 bit (a value column's dk entries side by side) and the convolution's last inputs, both zero at its
start, one pair per run of the layer; a step continues from what the request's earlier steps left, so a prompt may be cut anywhere.

q, k, v and b are one product; W_a1 and W_g1 are a second one, and W_a2 and W_g2 a third whose matrix has two blocks (zeros beside
them), so that decays and output gates come from one launch, in 32 bit.  Unit norms, decays, the recurrence and the norm behind it
are 32 bit whatever the compute type (``csrc/delta_rule.cu``): steps of single tokens and short portions take the tokens in turn
with the state in registers, long portions run in chunks of 32 tokens.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from . import linear
from .base import MIXERS, Mixer, StateSpec, TensorSpec
from .chunks import chunk_layout

PARALLEL_FROM = 33      # portions of at least this many tokens run in chunks
CONV_STATE = "conv"
STATE = "delta"


@MIXERS.register("channel_delta")
class ChannelDelta(Mixer):
    """Tensor names under ``prefix``: ``q``, ``k`` [G*dk, d], ``v`` [H*dv, d], each with ``<name>.conv`` [channels, taps]; ``b`` [H, d];
    ``A_log`` [H]; ``a1`` [decay_rank, d], ``a2`` [H*dk, decay_rank], ``dt_bias`` [H*dk]; ``g1`` [gate_rank, d], ``g2`` [H*dv, gate_rank];
    ``norm`` [dv]; ``o`` [d, H*dv]."""

    def __init__(self, prefix: str, width: int, heads: int, kv_heads: int, head_dim: int, value_dim: int, conv: int, decay_rank: int,
                 gate_rank: int, eps: float, guard: float = 1e-6):
        self.prefix, self.width = prefix, int(width)
        self.heads, self.kv_heads, self.dk, self.dv, self.taps = int(heads), int(kv_heads), int(head_dim), int(value_dim), int(conv)
        self.decay_rank, self.gate_rank = int(decay_rank), int(gate_rank)
        self.eps, self.guard = float(eps), float(guard)
        if self.heads % self.kv_heads:
            raise ValueError(f"{heads} heads are no multiple of {kv_heads} query/key heads")
        if self.taps < 1:
            raise ValueError("the convolution needs at least one tap")
        self.k_off = self.kv_heads * self.dk
        self.v_off = 2 * self.k_off
        self.channels = self.v_off + self.heads * self.dv
        self.w_in = self.w_low = self.w_up = self.w_o = self.conv_w = self.A_log = self.dt_bias = self.norm_w = None

    def tensor_specs(self):
        p, d, H, G, dk, dv = self.prefix, self.width, self.heads, self.kv_heads, self.dk, self.dv
        conv = lambda n, c: TensorSpec(p + n + ".conv", (c, self.taps), kind="vector", init="uniform:-0.5:0.5")      # noqa: E731
        return [TensorSpec(p + "q", (G * dk, d)), conv("q", G * dk), TensorSpec(p + "k", (G * dk, d)), conv("k", G * dk),
                TensorSpec(p + "v", (H * dv, d)), conv("v", H * dv), TensorSpec(p + "b", (H, d)),
                TensorSpec(p + "A_log", (H,), kind="vector", init="uniform:0:2"),
                TensorSpec(p + "a1", (self.decay_rank, d)), TensorSpec(p + "a2", (H * dk, self.decay_rank)),
                TensorSpec(p + "dt_bias", (H * dk,), kind="vector", init="uniform:-5:-1"),
                TensorSpec(p + "g1", (self.gate_rank, d)), TensorSpec(p + "g2", (H * dv, self.gate_rank)),
                TensorSpec(p + "norm", (dv,), kind="vector", init="norm"), TensorSpec(p + "o", (d, H * dv))]

    def bind(self, tensors):
        p = self.prefix
        f = lambda n: tensors[p + n].float().contiguous()   # noqa: E731  (what the recurrence reads is kept in 32 bit)
        self.w_in = linear.padded_rows(torch.cat([tensors[p + n] for n in ("q", "k", "v", "b")], dim=0))
        self.w_low = linear.padded_rows(torch.cat([tensors[p + "a1"], tensors[p + "g1"]], dim=0))
        a2, g2 = tensors[p + "a2"], tensors[p + "g2"]
        up = a2.new_zeros((a2.shape[0] + g2.shape[0], self.w_low.shape[0]))
        up[:a2.shape[0], :self.decay_rank] = a2
        up[a2.shape[0]:, self.decay_rank:self.decay_rank + self.gate_rank] = g2
        self.w_up = linear.padded_rows(up)
        self.w_o = tensors[p + "o"]
        self.conv_w = torch.cat([tensors[p + n + ".conv"].float() for n in ("q", "k", "v")], dim=0).contiguous()
        self.A_log, self.dt_bias = f("A_log"), f("dt_bias")
        self.norm_w = tensors[p + "norm"].float().repeat(self.heads).contiguous()

    def run_state_specs(self):
        return {CONV_STATE: StateSpec((max(self.taps - 1, 1), self.channels), torch.float32, 0.0),
                STATE: StateSpec((self.heads, self.dv, self.dk), torch.float32, 0.0)}

    def forward(self, ctx, x, cache):
        H, G, dk, dv = self.heads, self.kv_heads, self.dk, self.dv
        T = x.shape[0]
        st = cache.state
        rows = dict(row_slot=ctx.row_slot, row_q_start=ctx.row_q_start, row_q_len=ctx.row_q_len)
        src = linear.linear(ctx, x, self.w_in)                                  # [T, channels + H]: q | k | v | b
        qkv = torch.empty((T, self.channels), dtype=x.dtype, device=x.device)
        ops.conv_silu(src, src.shape[1], self.conv_w, None, st[CONV_STATE], qkv, tok_row=ctx.tok_row, single=ctx.decode_only, **rows)
        raw = linear.linear_f32(ctx, linear.linear(ctx, x, self.w_low), self.w_up)      # [T, H dk + H dv]: decays | gates
        o = torch.empty((T, H * dv), dtype=torch.float32, device=x.device)
        args = (qkv, self.k_off, self.v_off, src.data_ptr() + self.channels * src.element_size(), src.shape[1], raw, self.A_log, self.dt_bias,
                st[STATE], o)
        sizes = dict(H=H, G=G, dk=dk, dv=dv, q_scale=dk ** -0.5, guard=self.guard)
        if not ctx.replayable and ctx.max_q_len >= PARALLEL_FROM and ops.delta_rule_chunked_supported(dk, dv):
            base, total, most = chunk_layout(ctx, ops.delta_rule_chunk())
            per = H * ops.delta_rule_chunk_floats(dk, dv)
            bound = (-(-ctx.max_step_tokens // ops.delta_rule_chunk()) + ctx.max_rows) * per
            work = ctx.scratch("channel_delta.chunks", (total * per,), torch.float32, bound=(bound,))
            ops.delta_rule_chunked(*args, work, base, most, **sizes, **rows)
        else:
            if ctx.decode_only:
                rows["row_q_len"] = None
            ops.delta_rule(*args, **sizes, **rows)
        y = torch.empty((T, H * dv), dtype=x.dtype, device=x.device)
        ops.gated_rms_norm(o, raw.data_ptr() + H * dk * 4, raw.shape[1], self.norm_w, y, self.eps, group=dv, gate_dtype=torch.float32)
        return linear.linear(ctx, y, self.w_o)

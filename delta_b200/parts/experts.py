"""A mixture of experts: every token runs ``top`` of ``experts`` small gated feed-forwards, chosen by a router.

    z = W_router h                                   router logits, 32 bit
    the ``top`` largest z pick the experts; their weights are the softmax over the chosen logits only
    expert e:  y = act(W_gate,e h, W_up,e h),  W_down,e y          (the gated activation of ``clamped_glu``)
    out = sum over the chosen experts of weight * expert(h)  (+ sigmoid(w_sg . h) * shared(h) when there is a shared expert,
          a feed-forward of the same form that every token runs)
Nothing about the routing is read on the host: the (token, choice) pairs are sorted by expert on the device into tiles of
rows of one expert, and the two products of all experts are one launch each: warp-level MMA over tiles of 64 rows
(``csrc/experts.cu``), or, when a step brings many rows an expert, the tcgen05 product over tiles of 128 rows gathered side
by side (``csrc/gemm_tc.cu``).  The router's rows and
the shared expert's gate row are one matrix, so one product gives both.

Options: ``scoring`` "softmax_all": as "sigmoid" below with s = the softmax over all of the router's logits.  ``groups`` (count, keep): the
router's outputs form that many equal groups of neighbours; a group's score is the largest s + correction in it (``group_score`` "top2":
the sum of its two largest, or its only one), and only outputs of the ``keep`` best groups can be chosen.  ``identity`` n: the router has n more outputs than there are experts, the last ones; a token that
chooses one of them gets its own input h times the weight (no tensors, no product).  ``scoring`` "sigmoid": scores s = sigmoid(z); the ``top`` largest of s + correction (a tensor ``correction`` [E] when
``correction`` is set) are chosen, and the weights are the chosen s (without the correction) divided by their sum (+ 1e-20), times
``route_scale``; ``normalize`` False: the chosen s themselves, times ``route_scale``.  ``weight_input``: a choice's weight multiplies
what its expert reads, out = sum expert(weight * h), not what it gives: since (w h) W^T = w (h W^T), the first product's result is
multiplied by the weight before the activation (the tcgen05 path multiplies the rows as it gathers them).  ``shared`` {intermediate, limit, alpha, shift, gate}: ``gate`` False leaves the shared expert's sigmoid gate (and the
tensor ``shared.sg``) out, so it is added as it is.  ``activation`` "relu_squared": an expert is  W_down relu(W_up h)^2  with no gate branch.  ``wide_output``: the
weighted sum is handed on in 32 bit (for a 32-bit residual stream), not rounded to the compute type.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .base import FEED_FORWARDS, FeedForward, TensorSpec
from .feed_forward import ClampedGLU


TC_TILE = 128               # rows of a tile on the tcgen05 path
TC_ROWS_PER_EXPERT = 96     # from this many rows an expert on average, the products go to the tcgen05 kernel


@FEED_FORWARDS.register("experts")
class Experts(FeedForward):
    """Tensor names under ``prefix``: ``router`` [E, d]; ``e<i>.gate|up`` [F, d], ``e<i>.down`` [d, F]; with a shared expert
    ``shared.gate|up|down`` and ``shared.sg`` [1, d]."""

    def __init__(self, prefix: str, width: int, experts: int, top: int, intermediate: int, limit=None, alpha: float = 1.702,
                 shift: float = 1.0, shared: Optional[dict] = None, scoring: str = "softmax", correction: bool = False,
                 route_scale: float = 1.0, activation: str = "clamped_glu", wide_output: bool = False, normalize: bool = True,
                 weight_input: bool = False, identity: int = 0, groups: Optional[tuple] = None, group_score: str = "max"):
        self.prefix, self.width = prefix, int(width)
        self.experts, self.top, self.intermediate = int(experts), int(top), int(intermediate)
        self.identity, self.outputs = int(identity), int(experts) + int(identity)      # the router's outputs: experts, then identities
        self.groups = (int(groups[0]), int(groups[1])) if groups else None
        if group_score not in ops.GROUP_SCORES:
            raise ValueError(f"unknown score of a group '{group_score}' ({', '.join(ops.GROUP_SCORES)})")
        self.group_score = group_score
        if not (1 <= self.top <= self.outputs):
            raise ValueError(f"{self.top} of {self.experts} experts cannot be chosen")
        if limit is not None and float(limit) < 0:
            raise ValueError(f"a clamp at {limit} is no limit")
        self.limit, self.alpha, self.shift = (-1.0 if limit is None else float(limit)), float(alpha), float(shift)
        if scoring not in ops.ROUTER_SCORINGS:
            raise ValueError(f"unknown router scoring '{scoring}' ({', '.join(ops.ROUTER_SCORINGS)})")
        if self.groups and (scoring == "softmax" or self.outputs % self.groups[0] or not 1 <= self.groups[1] <= self.groups[0]
                            or self.groups[1] * (self.outputs // self.groups[0]) < self.top):
            raise ValueError(f"{self.groups[1]} of {self.groups[0]} groups of {self.outputs} experts do not hold {self.top} choices")
        if self.identity and (shared or weight_input):
            raise ValueError("identity experts beside a shared expert, or with weights on the experts' inputs, are not built")
        if activation not in ("clamped_glu", "relu_squared"):
            raise ValueError(f"unknown expert activation '{activation}' (clamped_glu, relu_squared)")
        if correction and scoring == "softmax":
            raise ValueError("a correction of the choice belongs to scores (sigmoid, softmax_all)")
        self.scoring, self.has_correction, self.route_scale = scoring, bool(correction), float(route_scale)
        self.gated = activation == "clamped_glu"
        self.wide_output = bool(wide_output)
        if self.wide_output and shared:
            raise ValueError("the 32-bit output is for experts without a shared expert (whose output has the compute type)")
        self.normalize, self.weight_input = bool(normalize), bool(weight_input)
        if not self.normalize and scoring == "softmax":
            raise ValueError("weights that are not normalised belong to scores (sigmoid, softmax_all)")
        self.correction = None
        self.shared = None
        self.shared_gate = bool(shared.get("gate", True)) if shared else False
        if shared:
            self.shared = ClampedGLU(prefix + "shared.", width, int(shared["intermediate"]), limit=shared.get("limit"),
                                     alpha=shared.get("alpha", alpha), shift=shared.get("shift", shift))
        self.w_router = self.w1 = self.w2 = None

    def tensor_specs(self):
        p, d, F = self.prefix, self.width, self.intermediate
        specs = [TensorSpec(p + "router", (self.outputs, d))]
        if self.has_correction:      # random weights: small beside the scores, which are about 1 / outputs each under a softmax over all
            spread = 0.2 if self.scoring == "sigmoid" else 0.2 / self.outputs
            specs.append(TensorSpec(p + "correction", (self.outputs,), kind="vector", init=f"uniform:{-spread}:{spread}"))
        for e in range(self.experts):
            specs += ([TensorSpec(f"{p}e{e}.gate", (F, d))] if self.gated else []) + [TensorSpec(f"{p}e{e}.up", (F, d)),
                                                                                     TensorSpec(f"{p}e{e}.down", (d, F))]
        if self.shared is not None:
            specs += self.shared.tensor_specs() + ([TensorSpec(p + "shared.sg", (1, d))] if self.shared_gate else [])
        return specs

    def bind(self, tensors):
        p = self.prefix
        rows = [tensors[p + "router"]] + ([tensors[p + "shared.sg"]] if self.shared_gate else [])
        self.w_router = torch.cat(rows, dim=0).contiguous()
        if self.gated:
            self.w1 = torch.stack([torch.cat([tensors[f"{p}e{e}.gate"], tensors[f"{p}e{e}.up"]], dim=0) for e in range(self.experts)]).contiguous()
        else:
            self.w1 = torch.stack([tensors[f"{p}e{e}.up"] for e in range(self.experts)]).contiguous()
        self.correction = tensors[p + "correction"].float().contiguous() if self.has_correction else None
        self.w2 = torch.stack([tensors[f"{p}e{e}.down"] for e in range(self.experts)]).contiguous()
        if self.shared is not None:
            self.shared.bind(tensors)

    def forward(self, ctx, x):
        T, d, E, top, F = x.shape[0], self.width, self.experts, self.top, self.intermediate
        dev, i32, f32 = x.device, torch.int32, torch.float32
        z = torch.empty((T, self.w_router.shape[0]), dtype=f32, device=dev)        # [T, E (+1)]
        choice = torch.empty((T, top), dtype=i32, device=dev)
        weight = torch.empty((T, top), dtype=f32, device=dev)
        ops.router(x, self.w_router, self.outputs, top, z, choice, weight, scoring=self.scoring, correction=self.correction, scale=self.route_scale,
                   normalize=self.normalize, groups=self.groups, group_score=self.group_score)
        act = "gated" if self.gated else "relu_squared"
        slots = T * top
        # weight_input: a slot's weight goes into the first product (or into the gathered rows), and the sum at the end has none
        row_scale = weight.view(-1) if self.weight_input else None
        # many rows an expert (prompt portions): tiles of 128 rows through the tcgen05 product; else tiles of 64 through warp-level MMA
        many = (x.dtype == torch.bfloat16 and "products" not in ctx.plain_kernels and slots >= TC_ROWS_PER_EXPERT * E and
                ops.experts_gemm_tc_supported(F, d, self.gated) and ops.experts_gemm_tc_supported(d, F, False))
        tile = TC_TILE if many else ops.experts_tile_rows()
        capacity = -(-(slots + (tile - 1) * min(E, slots)) // tile) * tile
        sorted_slots = torch.empty(capacity, dtype=i32, device=dev)
        tile_expert = torch.empty(capacity // tile, dtype=i32, device=dev)
        ops.experts_align(choice, E, sorted_slots, tile_expert, tile)
        y = torch.empty((capacity, F), dtype=x.dtype, device=dev)
        out_slots = torch.empty((slots, d), dtype=f32, device=dev)
        if many:
            rows = ops.experts_gather(x, sorted_slots, top, torch.empty((capacity, d), dtype=x.dtype, device=dev), row_scale=row_scale)
            ops.experts_gemm_tc(rows, self.w1, y, tile_expert, tile, n=F, glu=True if self.gated else act, limit=self.limit, alpha=self.alpha, shift=self.shift,
                                err=ctx.err)
            ops.experts_gemm_tc(y, self.w2, out_slots, tile_expert, tile, n=d, row_map=sorted_slots, err=ctx.err)
        else:
            ops.experts_gemm(x, self.w1, y, sorted_slots, tile_expert, top=top, n=F, k=d, act=act, limit=self.limit, alpha=self.alpha,
                             shift=self.shift, row_scale=row_scale)
            ops.experts_gemm(y, self.w2, out_slots, sorted_slots, tile_expert, top=top, n=d, k=F)
        out = torch.empty((T, d), dtype=f32 if self.wide_output else x.dtype, device=dev)     # wide: the weighted sum unrounded
        if self.weight_input:
            weight = None
        if self.shared is not None:
            s = self.shared.forward(ctx, x)
            ops.experts_combine(out_slots, weight, out, shared=s, gate_logit=(z.data_ptr() + self.outputs * 4) if self.shared_gate else None,
                                gate_stride=z.shape[1], top=top)
        else:      # a choice behind the experts' numbers is left out of the sorted tiles; the sum takes the input for it
            ops.experts_combine(out_slots, weight, out, top=top, identity=(x, choice, E) if self.identity else None)
        return out

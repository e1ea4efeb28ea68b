"""Burolorn as a ``ModelSpec``: a decoder whose config.json lists its layers.  Every layer is a pre-norm block on a 32-bit residual
stream with a token input behind the feed-forward,

    x <- x + attention(rms_norm1(x)),    x <- x + feed_forward(rms_norm2(x)),    x <- x + rms_norm_s(W_p (gelu(W_g x) * e))

(the second part may be absent), where e is the layer's own part of a second table's row of the token
(``parts/token_input.py``).  The mixer is grouped-query attention over chunks (``parts/row_attention.py``): queries, keys and values
go through short causal convolutions, queries and keys through an RMS norm per head and partly rotated positions; a query sees the
keys of its own chunk of positions; the softmax has a learned sink; values are mixed with those of the first layer of their group; the
heads' outputs are gated by one number per head.  The feed-forward is a dense silu-gated one or a mixture of experts by sigmoid
scores whose groups are ranked by their two largest scores, beside a gated shared expert (``parts/experts.py``).  The logits are
scaled.

Tensor names: ``embed``, ``side.embed``, ``head``, ``final.norm``; layer i: ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``,
``l<i>.side.*``.
"""
from __future__ import annotations

from typing import Optional

from ..config.burolorn_config import BurolornConfig
from ..config.engine_config import EngineConfig
from ..parts.base import PartSpec, TensorSpec
from ..parts.feed_forward import SILU_GATE
from .spec import LayerSpec, ModelSpec, RunEntry

VALUE_GROUP = "values"      # the model has one group of layers that mix values


def _mixer(cfg: BurolornConfig, i: int, max_pos: int) -> PartSpec:
    m, pre = cfg.layers[i].mixer, f"l{i}.mix."
    rot = m.get("rot") or None
    position = None
    if rot and rot["dims"]:
        position = PartSpec("rotary", dict(head_dim=rot["dims"], theta=rot["base"], max_positions=max_pos, interleaved=False), "position")
    mix = dict(group=VALUE_GROUP, first=i == cfg.first_mixing_layer) if m.get("v_mix") else None
    return PartSpec("sink_attention", dict(prefix=pre, width=cfg.width, heads=m["heads"], kv_heads=m["kv_heads"], head_dim=m["dim"],
                                           value_dim=m["vdim"], scale=m["scale"], position=position,
                                           rot_dims=rot["dims"] if position is not None else None, sink=True, qk_norm_eps=cfg.eps,
                                           conv=m.get("conv") or 0, chunk=(m.get("mask") or {}).get("size"), value_mix=mix,
                                           head_gate=True), "mixer")


def _feed_forward(cfg: BurolornConfig, i: int) -> Optional[PartSpec]:
    mlp, pre, d = cfg.layers[i].mlp, f"l{i}.mlp.", cfg.width
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("clamped_glu", dict(prefix=pre, width=d, intermediate=mlp["ff"], limit=None, **SILU_GATE), "feed_forward")
    r, shared = mlp["router"], mlp.get("shared")
    silu = dict(alpha=SILU_GATE["alpha"], shift=SILU_GATE["shift"])
    return PartSpec("experts", dict(prefix=pre, width=d, experts=r["experts"], top=r["top"], intermediate=mlp["expert"]["ff"], limit=None,
                                    shared=dict(intermediate=shared["ff"], limit=None, **silu) if shared else None, scoring="sigmoid",
                                    route_scale=float(r["scale"]) if r.get("scale") is not None else 1.0,
                                    groups=(r["groups"]["count"], r["groups"]["keep"]) if r.get("groups") else None, group_score="top2",
                                    **silu), "feed_forward")


def burolorn_spec(cfg: BurolornConfig, engine: Optional[EngineConfig] = None) -> ModelSpec:
    engine = engine or EngineConfig()
    d, n = cfg.width, len(cfg.layers)
    norm = lambda name: PartSpec("rms_norm", dict(name=name, width=d, eps=cfg.eps), "norm")     # noqa: E731
    layers, ignorable = [], []
    for i in range(n):
        parts = dict(norm1=norm(f"l{i}.norm1"), mixer=_mixer(cfg, i, engine.max_seq_len))
        ff = _feed_forward(cfg, i)
        if ff is not None:
            parts["norm2"] = norm(f"l{i}.norm2")
            parts["feed_forward"] = ff
        else:
            ignorable.append(f"l{i}.norm2")
        if cfg.side_dim:
            parts["token_input"] = PartSpec("table_gate", dict(prefix=f"l{i}.side.", table="side.embed", vocab=cfg.vocab, width=d,
                                                               dim=cfg.side_dim, index=i, parts=n, eps=cfg.eps), "token_input")
        layers.append(LayerSpec(parts, block="residual_pre_norm"))
    if cfg.first_mixing_layer is not None:
        ignorable.append(f"l{cfg.first_mixing_layer}.mix.vmix")      # stored, although the group's first layer mixes nothing in
    return ModelSpec(
        vocab_size=cfg.vocab, width=d, layers=tuple(layers), order=tuple(RunEntry(i) for i in range(n)), final_norm=norm("final.norm"),
        embedding=TensorSpec("embed", (cfg.vocab, d), kind="table"), lm_head=TensorSpec("head", (cfg.vocab, d), kind="matrix"),
        max_positions=engine.max_seq_len, stream=PartSpec("residual_f32", dict(width=d), "stream"), logit_scale=cfg.logit_scale,
        ignorable_tensors=tuple(ignorable))

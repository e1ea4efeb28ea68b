"""Vazunex as a ``ModelSpec``: a decoder whose config.json lists its layers.  The embedding goes through a norm of its own; every
layer is a pre-norm block on a 32-bit residual stream whose sublayer outputs are multiplied by one constant m,

    x <- x + m mixer(rms_norm1(x)),    x <- x + m experts(rms_norm2(x))        (the second half may be absent)

with RMS norms whose stored weight is the deviation from one.  The mixers:

  * ``channel_delta``: a gated delta rule with a decay per head and key channel behind short convolutions
    (``parts/channel_delta.py``);
  * ``mamba2``: a state-space recurrence with one decay per head (``parts/state_space.py``);
  * ``latent_attention``: keys and values through a small latent, a short rotated key part that all heads share, a sliding window, a
    learned sink and an output gate (``parts/latent_attention.py``).

The feed-forward is a mixture of silu-gated experts: softmax scores over all of the router's outputs, a correction that enters the
choice only, groups of neighbours of which the best are kept, weights that are not normalised, and outputs that stand for no expert
but for the layer's own input (``parts/experts.py``).  The logits are scaled.

Tensor names: ``embed``, ``embed.norm``, ``head``, ``final.norm``; layer i: ``l<i>.norm1|norm2``, ``l<i>.mix.*``, ``l<i>.mlp.*``.
"""
from __future__ import annotations

from typing import Optional

from ..config.engine_config import EngineConfig
from ..config.vazunex_config import VazunexConfig
from ..parts.base import PartSpec, TensorSpec
from ..parts.feed_forward import SILU_GATE
from .spec import LayerSpec, ModelSpec, RunEntry

UNIT_GUARD = 1e-6       # added to the sum of squares when queries and keys of the delta rule are made unit vectors
WEIGHT_OFFSET = 1.0     # the norms store their weight's deviation from one


def _mixer(cfg: VazunexConfig, i: int, max_pos: int) -> PartSpec:
    L = cfg.layers[i]
    m, pre, d = L.mixer, f"l{i}.mix.", cfg.width
    if L.type == "channel_delta":
        return PartSpec("channel_delta", dict(prefix=pre, width=d, heads=m["heads"], kv_heads=m["kv_heads"], head_dim=m["dim"],
                                              value_dim=m["vdim"], conv=m["conv"], decay_rank=m["decay_rank"], gate_rank=m["gate_rank"],
                                              eps=cfg.eps, guard=UNIT_GUARD), "mixer")
    if L.type == "mamba2":
        return PartSpec("state_space", dict(prefix=pre, width=d, heads=m["heads"], head_dim=m["vdim"], state=m["state"], groups=m["groups"],
                                            conv=m["conv"], norm_groups=m["norm_groups"], eps=cfg.eps), "mixer")
    position = None
    if m["rot_dim"]:
        position = PartSpec("rotary", dict(head_dim=m["rot"]["dims"], theta=m["rot"]["base"], max_positions=max_pos, interleaved=False), "position")
    return PartSpec("latent_attention", dict(prefix=pre, width=d, heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"],
                                             value_dim=m["vdim"], kv_rank=m["kv_rank"], eps=cfg.eps, scale=m["scale"], position=position,
                                             rot_dims=m["rot"]["dims"] if m["rot_dim"] else None,
                                             window=(m.get("mask") or {}).get("size"), sink=True, gate=True), "mixer")


def _feed_forward(cfg: VazunexConfig, i: int) -> Optional[PartSpec]:
    mlp, pre, d = cfg.layers[i].mlp, f"l{i}.mlp.", cfg.width
    if mlp is None:
        return None
    r = mlp["router"]
    groups = (r["groups"]["count"], r["groups"]["keep"]) if r.get("groups") else None
    return PartSpec("experts", dict(prefix=pre, width=d, experts=r["experts"], top=r["top"], intermediate=mlp["expert"]["ff"], limit=None,
                                    alpha=SILU_GATE["alpha"], shift=SILU_GATE["shift"], scoring="softmax_all", correction=True,
                                    route_scale=float(r["scale"]) if r.get("scale") is not None else 1.0, normalize=False,
                                    identity=int(r.get("identity") or 0), groups=groups, wide_output=True), "feed_forward")


def vazunex_spec(cfg: VazunexConfig, engine: Optional[EngineConfig] = None) -> ModelSpec:
    engine = engine or EngineConfig()
    d = cfg.width
    norm = lambda name: PartSpec("rms_norm", dict(name=name, width=d, eps=cfg.eps, weight_offset=WEIGHT_OFFSET), "norm")     # noqa: E731
    layers = []
    for i in range(len(cfg.layers)):
        parts = dict(norm1=norm(f"l{i}.norm1"), mixer=_mixer(cfg, i, engine.max_seq_len))
        ff = _feed_forward(cfg, i)
        if ff is not None:
            parts["norm2"] = norm(f"l{i}.norm2")
            parts["feed_forward"] = ff
        layers.append(LayerSpec(parts, block="residual_pre_norm", options=dict(update_scale=cfg.residual_mult)))
    return ModelSpec(
        vocab_size=cfg.vocab, width=d, layers=tuple(layers), order=tuple(RunEntry(i) for i in range(len(layers))), final_norm=norm("final.norm"),
        embedding=TensorSpec("embed", (cfg.vocab, d), kind="table"), lm_head=TensorSpec("head", (cfg.vocab, d), kind="matrix"),
        max_positions=engine.max_seq_len, stream=PartSpec("residual_f32", dict(width=d, start_norm=norm("embed.norm")), "stream"),
        logit_scale=cfg.logit_scale)

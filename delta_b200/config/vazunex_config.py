"""Typed configuration of the Vazunex design, read from its config.json.

The file names the design in ``architecture`` and gives every size and every constant that may differ between
models of the design:

    vocab, width                         token interface and stream width
    norm.eps                             eps of every RMS norm (stream norms, the norms inside the mixers)
    residual_mult                        constant on every sublayer's output (absent: 1)
    logit_scale                          factor on the logits (absent: 1)
    layers[i] {type, mixer, mlp}         the mixer's kind and sizes; mlp or null

Mixer kinds and their keys:
    channel_delta      heads, kv_heads, dim, vdim, conv; decay_rank and gate_rank (the rows of the tensors ``a1`` and ``g1``; absent:
                       taken from the tensors' shapes in the model folder)
    mamba2             heads, vdim, state, groups, conv, norm_groups
    latent_attention   heads, dim, rot_dim, vdim, kv_rank, scale, mask {size} (absent: every earlier token is seen),
                       rot {base, dims} (needed when rot_dim > 0)
Feed-forward kinds (``kind``; absent: moe):
    moe         router {experts, top, identity (absent: 0), groups {count, keep} (absent: no groups), scale (absent: 1)}, expert {ff}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .model_config import ConfigError

MIXER_KEYS = {
    "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
    "mamba2": ("heads", "vdim", "state", "groups", "conv", "norm_groups"),
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"),
}
RANKS = {"decay_rank": "a1", "gate_rank": "g1"}      # sizes that config.json may leave to the shapes of these tensors


@dataclass(frozen=True)
class VazunexLayer:
    type: str
    mixer: dict
    mlp: Optional[dict]


def rank_tensor(layer: int, key: str) -> str:
    return f"l{layer}.mix.{RANKS[key]}"


def sizes_from_shapes(c: dict, shapes: dict) -> dict:
    """config.json with the sizes that only the tensors give filled in: the ranks of every delta layer's decay and gate projections."""
    out = dict(c)
    layers = []
    for i, L in enumerate(c.get("layers") or []):
        m = L.get("mixer") if isinstance(L, dict) else None
        if isinstance(m, dict) and L.get("type") == "channel_delta":
            found = {k: int(shapes[rank_tensor(i, k)][0]) for k in RANKS if m.get(k) is None and rank_tensor(i, k) in shapes}
            L = dict(L, mixer=dict(m, **found))
        layers.append(L)
    out["layers"] = layers
    return out


@dataclass(frozen=True)
class VazunexConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    layers: tuple
    residual_mult: float = 1.0
    logit_scale: float = 1.0

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def from_dict(c: dict) -> "VazunexConfig":
        def need(d, key, where):
            if not isinstance(d, dict) or key not in d or d[key] is None:
                raise ConfigError(f"config.json has no '{key}' in {where}")
            return d[key]

        raw_layers = need(c, "layers", "the model")
        if not raw_layers:
            raise ConfigError("config.json lists no layers")
        layers = []
        for i, L in enumerate(raw_layers):
            kind = need(L, "type", f"layer {i}")
            if kind not in MIXER_KEYS:
                raise ConfigError(f"layer {i}: unknown mixer type '{kind}'; known: {', '.join(MIXER_KEYS)}")
            m = dict(need(L, "mixer", f"layer {i}"))
            for k in MIXER_KEYS[kind]:
                need(m, k, f"the mixer of layer {i}")
            if kind == "channel_delta":
                for k in RANKS:
                    need(m, k, f"the mixer of layer {i} (nor is there a tensor '{rank_tensor(i, k)}' to take it from)")
            if kind == "latent_attention":
                if m["rot_dim"]:
                    rot = need(m, "rot", f"the mixer of layer {i}")
                    need(rot, "base", f"rot of layer {i}")
                    need(rot, "dims", f"rot of layer {i}")
                if m.get("mask"):
                    need(m["mask"], "size", f"mask of layer {i}")
            mlp = L.get("mlp")
            if mlp is not None:
                mlp = dict(mlp)
                mk = mlp.get("kind") or "moe"      # the design has one kind of feed-forward
                if mk != "moe":
                    raise ConfigError(f"layer {i}: unknown feed-forward kind '{mk}' (moe)")
                r = need(mlp, "router", f"mlp of layer {i}")
                need(r, "experts", f"router of layer {i}")
                need(r, "top", f"router of layer {i}")
                if r.get("groups"):
                    need(r["groups"], "count", f"router.groups of layer {i}")
                    need(r["groups"], "keep", f"router.groups of layer {i}")
                need(need(mlp, "expert", f"mlp of layer {i}"), "ff", f"expert of layer {i}")
            layers.append(VazunexLayer(kind, m, mlp))

        def number(key):
            return float(c[key]) if c.get(key) is not None else 1.0

        cfg = VazunexConfig(
            architecture=str(c.get("architecture") or (c.get("architectures") or ["Vazunex"])[0]),
            vocab=int(need(c, "vocab", "the model")), width=int(need(c, "width", "the model")),
            eps=float(need(need(c, "norm", "the model"), "eps", "norm")), layers=tuple(layers),
            residual_mult=number("residual_mult"), logit_scale=number("logit_scale"))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab < 1 or self.width < 1:
            raise ConfigError("vocab and width must be positive")
        for i, L in enumerate(self.layers):
            m = L.mixer
            if L.type == "channel_delta":
                if min(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], m["decay_rank"], m["gate_rank"]) < 1:
                    raise ConfigError(f"layer {i}: heads, kv_heads, dim, vdim, conv and the ranks must be positive")
                if m["heads"] % m["kv_heads"]:
                    raise ConfigError(f"layer {i}: {m['heads']} heads are no multiple of {m['kv_heads']} query/key heads")
            elif L.type == "mamba2":
                if min(m["heads"], m["vdim"], m["state"], m["groups"], m["conv"], m["norm_groups"]) < 1:
                    raise ConfigError(f"layer {i}: heads, vdim, state, groups, conv and norm_groups must be positive")
                if m["heads"] % m["groups"]:
                    raise ConfigError(f"layer {i}: {m['heads']} heads are no multiple of {m['groups']} groups")
                if (m["heads"] * m["vdim"]) % m["norm_groups"]:
                    raise ConfigError(f"layer {i}: {m['heads'] * m['vdim']} channels do not split into {m['norm_groups']} equal parts")
            else:
                if min(m["heads"], m["dim"], m["vdim"], m["kv_rank"]) < 1 or m["rot_dim"] < 0:
                    raise ConfigError(f"layer {i}: heads, dim, vdim and kv_rank must be positive")
                if m["rot_dim"]:
                    dims = int(m["rot"]["dims"])
                    if dims % 2 or dims > m["rot_dim"] or dims < 2:
                        raise ConfigError(f"layer {i}: rot.dims {dims} must be even and at most rot_dim {m['rot_dim']}")
                if m.get("mask") and int(m["mask"]["size"]) < 1:
                    raise ConfigError(f"layer {i}: a window of {m['mask']['size']} tokens sees nothing")
            if L.mlp:
                r = L.mlp["router"]
                outputs = int(r["experts"]) + int(r.get("identity") or 0)
                if int(r["experts"]) < 1 or int(r.get("identity") or 0) < 0 or not (1 <= r["top"] <= outputs):
                    raise ConfigError(f"layer {i}: top {r['top']} of {r['experts']} experts and {r.get('identity') or 0} identities")
                if r.get("groups"):
                    count, keep = int(r["groups"]["count"]), int(r["groups"]["keep"])
                    if count < 1 or outputs % count or not (1 <= keep <= count) or keep * (outputs // count) < r["top"]:
                        raise ConfigError(f"layer {i}: {keep} of {count} groups of {outputs} router outputs do not hold {r['top']} choices")

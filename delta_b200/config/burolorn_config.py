"""Typed configuration of the Burolorn design, read from its config.json.

The file names the design in ``architecture`` and gives every size and every constant that may differ between
models of the design:

    vocab, width                         token interface and stream width
    norm.eps                             eps of every RMS norm (stream norms, query and key norms, token-input norms)
    token_side {dim}                     size of a layer's token input (absent: no layer has one)
    logit_scale                          factor on the logits (absent: 1)
    layers[i] {type, mixer, mlp}         the mixer's kind and sizes; mlp or null

Mixer kinds and their keys:
    attention   heads, kv_heads, dim, vdim, scale, conv (taps; absent: no convolution), rot {base, dims} (absent: no rotation),
                mask {size} (chunk length; absent: every earlier token is seen), v_mix (absent: false)
Feed-forward kinds:
    dense       ff
    moe         router {experts, top, groups {count, keep} (absent: no groups), scale (absent: 1)}, expert {ff},
                shared {ff} (absent: no shared expert)
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .model_config import ConfigError

MIXER_KEYS = {"attention": ("heads", "kv_heads", "dim", "vdim", "scale")}


@dataclass(frozen=True)
class BurolornLayer:
    type: str
    mixer: dict
    mlp: Optional[dict]


@dataclass(frozen=True)
class BurolornConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    layers: tuple
    side_dim: int = 0
    logit_scale: float = 1.0

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def first_mixing_layer(self) -> Optional[int]:
        """The layer whose values the later layers of the value-mixing group mix in (None: no layer mixes)."""
        return next((i for i, L in enumerate(self.layers) if L.mixer.get("v_mix")), None)

    @staticmethod
    def from_dict(c: dict) -> "BurolornConfig":
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
            if m.get("rot"):
                need(m["rot"], "base", f"rot of layer {i}")
                need(m["rot"], "dims", f"rot of layer {i}")
            if m.get("mask"):
                need(m["mask"], "size", f"mask of layer {i}")
            mlp = L.get("mlp")
            if mlp is not None:
                mlp = dict(mlp)
                mk = need(mlp, "kind", f"mlp of layer {i}")
                if mk == "dense":
                    need(mlp, "ff", f"mlp of layer {i}")
                elif mk == "moe":
                    r = need(mlp, "router", f"mlp of layer {i}")
                    need(r, "experts", f"router of layer {i}")
                    need(r, "top", f"router of layer {i}")
                    if r.get("groups"):
                        need(r["groups"], "count", f"router.groups of layer {i}")
                        need(r["groups"], "keep", f"router.groups of layer {i}")
                    need(need(mlp, "expert", f"mlp of layer {i}"), "ff", f"expert of layer {i}")
                    if mlp.get("shared"):
                        need(mlp["shared"], "ff", f"shared expert of layer {i}")
                else:
                    raise ConfigError(f"layer {i}: unknown feed-forward kind '{mk}' (dense, moe)")
            layers.append(BurolornLayer(kind, m, mlp))
        side = c.get("token_side")
        cfg = BurolornConfig(
            architecture=str(c.get("architecture") or (c.get("architectures") or ["Burolorn"])[0]),
            vocab=int(need(c, "vocab", "the model")), width=int(need(c, "width", "the model")),
            eps=float(need(need(c, "norm", "the model"), "eps", "norm")), layers=tuple(layers),
            side_dim=int(need(side, "dim", "token_side")) if side else 0,
            logit_scale=float(c["logit_scale"]) if c.get("logit_scale") is not None else 1.0)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab < 1 or self.width < 1:
            raise ConfigError("vocab and width must be positive")
        if self.side_dim < 0:
            raise ConfigError(f"token_side.dim {self.side_dim} is no size")
        first = self.first_mixing_layer
        for i, L in enumerate(self.layers):
            m = L.mixer
            if min(m["heads"], m["kv_heads"], m["dim"], m["vdim"]) < 1 or (m.get("conv") is not None and m["conv"] < 0):
                raise ConfigError(f"layer {i}: heads, kv_heads, dim and vdim must be positive")
            if m["heads"] % m["kv_heads"]:
                raise ConfigError(f"layer {i}: {m['heads']} heads are no multiple of {m['kv_heads']} key-value heads")
            rot = m.get("rot")
            if rot and (rot["dims"] % 2 or not 0 <= rot["dims"] <= m["dim"]):
                raise ConfigError(f"layer {i}: rot.dims {rot['dims']} must be even and at most dim {m['dim']}")
            if m.get("mask") and int(m["mask"]["size"]) < 1:
                raise ConfigError(f"layer {i}: a chunk of {m['mask']['size']} tokens holds nothing")
            if m.get("v_mix"):
                f = self.layers[first].mixer
                if m["kv_heads"] * m["vdim"] != f["kv_heads"] * f["vdim"]:
                    raise ConfigError(f"layer {i}: {m['kv_heads']} x {m['vdim']} values cannot be mixed with the {f['kv_heads']} x {f['vdim']} "
                                      f"of layer {first}")
            if L.mlp and L.mlp["kind"] == "moe":
                r = L.mlp["router"]
                if not (1 <= r["top"] <= r["experts"]):
                    raise ConfigError(f"layer {i}: top {r['top']} of {r['experts']} experts")
                if r.get("groups"):
                    count, keep = int(r["groups"]["count"]), int(r["groups"]["keep"])
                    if count < 1 or r["experts"] % count or not (1 <= keep <= count) or keep * (r["experts"] // count) < r["top"]:
                        raise ConfigError(f"layer {i}: {keep} of {count} groups of {r['experts']} experts do not hold {r['top']} choices")

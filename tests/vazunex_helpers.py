"""Small Vazunex configurations and weights for the tests.  Tensor names and shapes are written out here from the
configuration, independently of the engine's own list, so a name or shape the engine gets wrong shows as a loading
error."""
from __future__ import annotations

import math

import torch

from roletar_helpers import write_folder  # noqa: F401  (the folder writer knows no design)


def delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    # the ranks are not in config.json (the tensors' shapes say them); taken out by ``strip``
    return dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, _ranks=(decay_rank, gate_rank)))


def ssd(heads, vdim, state, groups, conv, norm_groups):
    return dict(type="mamba2", mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups))


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, window=None, base=10000.0):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale)
    if rot_dim:
        m["rot"] = dict(base=base, dims=rot_dim)
    if window is not None:
        m["mask"] = dict(size=window)
    return dict(type="latent_attention", mixer=m)


def moe(layer, experts, top, ff, identity=None, groups=None, scale=None):
    r = dict(experts=experts, top=top)
    if identity is not None:
        r["identity"] = identity
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    if scale is not None:
        r["scale"] = scale
    return dict(layer, mlp=dict(kind="moe", router=r, expert=dict(ff=ff)))


def bare(layer):
    return dict(layer, mlp=None)


def _named(which: str) -> dict:
    base = dict(architecture="Vazunex", norm=dict(eps=1e-5))
    if which == "mix":      # every mixer; groups, identities and neither; shared query/key heads and maps; layers without feed-forward
        return dict(base, vocab=300, width=96, logit_scale=0.7, residual_mult=0.4, layers=[
            moe(ssd(6, 16, 24, 2, 4, 3), 7, 3, 40, identity=2, groups=(3, 2), scale=1.7),
            bare(latent(3, 16, 8, 24, 40, 0.2, window=21, base=1000.0)),
            moe(delta(6, 3, 16, 24, 4, 12, 20), 5, 2, 24, identity=1, groups=(2, 1), scale=2.5),
            moe(latent(2, 24, 16, 16, 24, 0.15, window=50, base=50.0), 6, 2, 32, scale=1.3),
            moe(ssd(4, 40, 12, 4, 2, 1), 4, 2, 24, identity=4, groups=(4, 3)),
            bare(delta(4, 1, 24, 16, 3, 8, 8))])
    if which == "odd":      # no size a multiple of 4; pages of two tokens; a window of five
        return dict(base, vocab=61, width=50, norm=dict(eps=1e-6), logit_scale=1.3, residual_mult=0.9, layers=[
            moe(delta(3, 1, 10, 6, 2, 5, 7), 5, 3, 9, identity=1, groups=(3, 2), scale=0.6),
            moe(latent(3, 6, 6, 10, 14, 0.3, window=5, base=300.0), 3, 2, 11, identity=2),
            moe(ssd(3, 14, 9, 1, 5, 6), 6, 1, 10, identity=3, groups=(9, 4), scale=3.0),
            bare(delta(2, 2, 7, 11, 6, 3, 2))])
    if which == "one":      # what other models make larger is 1 or absent here: heads, groups, experts, taps, a window of one token,
        return dict(base, vocab=128, width=48, layers=[     # no multiplier, no scale, no groups, no identities
            moe(ssd(1, 8, 1, 1, 1, 1), 1, 1, 20), moe(delta(1, 1, 8, 8, 1, 1, 1), 2, 2, 16),
            moe(latent(1, 8, 2, 8, 12, 0.4, window=1, base=10.0), 1, 1, 12, identity=1), bare(latent(2, 12, 4, 8, 10, 0.5))])
    if which == "sharp":    # no experts (nothing hangs on a close call): single keys carry most of the weight; windows at page borders
        return dict(base, vocab=97, width=64, norm=dict(eps=1e-2), logit_scale=0.5, residual_mult=0.7, layers=[
            bare(latent(4, 16, 8, 16, 24, 0.5, window=16, base=100.0)), bare(delta(4, 2, 16, 32, 4, 16, 16)), bare(ssd(4, 32, 16, 1, 4, 2)),
            bare(latent(2, 32, 8, 8, 16, 0.3, window=33)), bare(delta(2, 2, 32, 16, 4, 8, 8))])
    if which == "wide":     # sizes that the tensor-core kernels take (multiples of 16 and 64)
        return dict(base, vocab=200, width=128, logit_scale=0.8, residual_mult=0.6, layers=[
            moe(delta(4, 2, 64, 32, 4, 32, 32), 6, 2, 64, identity=2, groups=(4, 2), scale=1.5),
            moe(latent(4, 32, 32, 32, 64, 0.12, window=100, base=5000.0), 4, 2, 64, identity=1),
            moe(ssd(8, 32, 64, 2, 4, 2), 3, 1, 128, identity=1, groups=(2, 1))])
    if which == "larger":   # widths, heads and experts that the tcgen05 products and the chunked kernels take in long portions
        return dict(base, vocab=1000, width=512, logit_scale=0.6, residual_mult=0.5, layers=[
            moe(ssd(16, 64, 128, 2, 4, 1), 6, 2, 256, identity=2, groups=(2, 1), scale=2.0),
            moe(delta(4, 2, 128, 128, 4, 64, 64), 8, 2, 256, scale=1.5),
            moe(latent(8, 64, 32, 64, 128, 0.1, window=300, base=100000.0), 7, 2, 256, identity=1, groups=(4, 2))])
    if which == "only_delta":
        return dict(base, vocab=97, width=40, layers=[bare(delta(4, 2, 16, 8, 4, 6, 10))])
    if which == "only_ssd":
        return dict(base, vocab=97, width=40, layers=[bare(ssd(4, 16, 20, 2, 3, 2))])
    if which == "only_latent":
        return dict(base, vocab=97, width=40, layers=[bare(latent(2, 16, 8, 12, 20, 0.3, window=13, base=100.0))])
    if which == "only_experts":     # the mixer is tiny, the feed-forward dominates
        return dict(base, vocab=97, width=40, layers=[moe(latent(1, 4, 2, 4, 6, 0.5, window=3), 7, 3, 24, identity=2, groups=(3, 2), scale=1.5),
                                                      moe(ssd(1, 4, 2, 1, 2, 1), 4, 2, 12, identity=2, groups=(2, 1))])
    raise KeyError(which)


PAGE_SIZE = {"larger": 16, "wide": 16, "mix": 16, "odd": 2, "one": 4, "sharp": 16, "only_delta": 8, "only_ssd": 8, "only_latent": 4, "only_experts": 16}


def strip(cfg: dict) -> dict:
    """config.json as a model folder holds it: the ranks are left to the tensors' shapes."""
    return dict(cfg, layers=[dict(L, mixer={k: v for k, v in L["mixer"].items() if k != "_ranks"}) for L in cfg["layers"]])


def config(which: str) -> dict:
    return strip(_named(which))


def make_weights(cfg: dict, seed: int) -> dict:
    """name -> float32 tensor whose values are all representable in bfloat16; ``cfg`` with the ranks (``_named``)."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]

    def mat(out, inp, gain=1.0):
        return torch.randn(out, inp, generator=g) * (gain / math.sqrt(inp))

    def uni(shape, a, b):
        return a + (b - a) * torch.rand(shape, generator=g)

    W = {"embed": torch.randn(cfg["vocab"], d, generator=g), "embed.norm": uni((d,), -0.2, 0.2), "head": mat(cfg["vocab"], d, 2.0),
         "final.norm": uni((d,), -0.2, 0.2)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        W[p + "norm1"] = uni((d,), -0.2, 0.2)
        if L["type"] == "channel_delta":
            H, G, dk, dv, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            ra, rg = m["_ranks"]
            for n, c in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                W[q + n], W[q + n + ".conv"] = mat(c, d, 1.5), uni((c, taps), -0.8, 0.8)
            W[q + "b"], W[q + "A_log"], W[q + "dt_bias"] = mat(H, d, 1.5), uni((H,), -2.0, 2.0), uni((H * dk,), -6.0, 0.0)
            W[q + "a1"], W[q + "a2"] = mat(ra, d, 1.0), mat(H * dk, ra, 1.0)
            W[q + "g1"], W[q + "g2"] = mat(rg, d, 1.5), mat(H * dv, rg, 1.5)
            W[q + "norm"], W[q + "o"] = uni((dv,), 0.7, 1.3), mat(d, H * dv, 2.0)
        elif L["type"] == "mamba2":
            H, P, N, G, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
            inner, ch = H * P, H * P + 2 * G * N
            W[q + "in"], W[q + "conv"], W[q + "conv.b"] = mat(inner + ch + H, d, 1.5), uni((ch, taps), -0.8, 0.8), uni((ch,), -0.2, 0.2)
            W[q + "dt_bias"], W[q + "A_log"], W[q + "D"] = uni((H,), -5.0, 0.5), uni((H,), -2.0, 2.0), uni((H,), 0.5, 1.5)
            W[q + "norm"], W[q + "o"] = uni((inner,), 0.7, 1.3), mat(d, inner, 2.0)
        else:
            H, dk, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            W[q + "q"], W[q + "dkv"], W[q + "dkv.norm"] = mat(H * (dk + dr), d, 2.0), mat(R + dr, d, 2.0), uni((R,), 0.8, 1.2)
            W[q + "uk"], W[q + "uv"], W[q + "o"] = mat(H * dk, R, 2.0), mat(H * dv, R, 1.5), mat(d, H * dv, 2.0)
            W[q + "sink"], W[q + "g"] = uni((H,), -1.0, 3.0), mat(H * dv, d, 1.5)
        mlp = L.get("mlp")
        if not mlp:
            continue
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        outputs = E + (mlp["router"].get("identity") or 0)
        W[p + "norm2"], W[p + "mlp.router"] = uni((d,), -0.2, 0.2), mat(outputs, d, 3.0)
        W[p + "mlp.correction"] = uni((outputs,), -0.6, 0.1)      # mostly negative choice scores
        for e in range(E):
            W[f"{p}mlp.e{e}.gate"], W[f"{p}mlp.e{e}.up"], W[f"{p}mlp.e{e}.down"] = mat(ff, d, 1.5), mat(ff, d, 1.5), mat(d, ff)
    return {k: v.to(torch.bfloat16).float() for k, v in W.items()}


def build(which: str, seed: int):
    """(config.json's dict, weights) of a named test model."""
    full = _named(which)
    return strip(full), make_weights(full, seed)

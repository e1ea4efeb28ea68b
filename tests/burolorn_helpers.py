"""Small Burolorn configurations and weights for the tests.  Tensor names and shapes are written out here from the
configuration, independently of the engine's own list, so a name or shape the engine gets wrong shows as a loading
error."""
from __future__ import annotations

import math

import torch

from roletar_helpers import write_folder  # noqa: F401  (the folder writer knows no design)


def attention(heads, kv_heads, dim, vdim, scale, conv=4, chunk=None, rot=None, v_mix=True):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, v_mix=v_mix)
    if conv:
        m["conv"] = conv
    if chunk is not None:
        m["mask"] = dict(size=chunk)
    if rot is not None:
        m["rot"] = dict(dims=rot[0], base=rot[1])
    return dict(type="attention", mixer=m)


def dense(layer, ff):
    return dict(layer, mlp=dict(kind="dense", ff=ff))


def moe(layer, experts, top, ff, shared=None, groups=None, scale=None):
    r = dict(experts=experts, top=top)
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    if scale is not None:
        r["scale"] = scale
    mlp = dict(kind="moe", router=r, expert=dict(ff=ff))
    if shared:
        mlp["shared"] = dict(ff=shared)
    return dict(layer, mlp=mlp)


def bare(layer):
    return dict(layer, mlp=None)


def config(which: str) -> dict:
    base = dict(architecture="Burolorn", norm=dict(eps=1e-5))
    if which == "mix":      # every option: chunks of two lengths and none, groups of three sizes and none, layers that mix no values (the
        return dict(base, vocab=300, width=96, logit_scale=0.7, token_side=dict(dim=20), layers=[     # first one too), no feed-forward
            dense(attention(6, 3, 16, 24, 0.3, conv=4, chunk=24, rot=(8, 1000.0), v_mix=False), 40),
            moe(attention(4, 2, 32, 16, 0.2, conv=3, chunk=50, rot=(32, 500.0)), 6, 3, 24, shared=40, groups=(3, 2), scale=1.7),
            bare(attention(4, 4, 16, 8, 0.25, conv=2, rot=(6, 50.0))),
            moe(attention(2, 1, 24, 32, 0.2, conv=4, chunk=24), 8, 2, 32, groups=(2, 1), scale=2.5),
            moe(attention(8, 2, 16, 16, 0.3, conv=0, chunk=50, rot=(16, 100.0)), 5, 2, 16, shared=16),
            dense(attention(6, 3, 16, 24, 0.3, conv=4, chunk=24, rot=(8, 1000.0), v_mix=False), 24)])
    if which == "odd":      # no size a multiple of 4; pages of two tokens; chunks of five; more taps than any vector kernel takes
        return dict(base, vocab=61, width=50, norm=dict(eps=1e-6), logit_scale=1.3, token_side=dict(dim=7), layers=[
            moe(attention(3, 1, 11, 6, 0.4, conv=5, chunk=5, rot=(6, 300.0)), 9, 4, 9, shared=11, groups=(3, 2), scale=0.6),
            dense(attention(3, 3, 10, 2, 0.3, conv=6, chunk=17, rot=(2, 30.0)), 13),
            moe(attention(2, 2, 7, 3, 0.3, conv=2), 3, 1, 10, groups=(3, 2))])
    if which == "one":      # what other models make larger is 1 or absent here: heads, taps, experts, groups; a chunk of one token;
        return dict(base, vocab=128, width=48, layers=[     # no token inputs, no scales, no rotation, no shared expert
            moe(attention(1, 1, 8, 8, 0.5, conv=1, chunk=1), 1, 1, 20), dense(attention(1, 1, 2, 4, 0.7, conv=1, rot=(2, 10.0), v_mix=False), 16),
            moe(attention(2, 1, 16, 8, 0.3, conv=2), 2, 2, 16, groups=(1, 1))])
    if which == "sharp":    # no experts (nothing hangs on a close call): single keys carry most of the weight; chunks at page borders
        return dict(base, vocab=97, width=64, norm=dict(eps=1e-2), logit_scale=0.5, token_side=dict(dim=16), layers=[
            dense(attention(4, 2, 16, 16, 1.0, conv=4, chunk=16, rot=(8, 100.0)), 48), bare(attention(2, 2, 32, 16, 0.6, conv=4, chunk=33, rot=(32, 1e4))),
            dense(attention(4, 1, 16, 32, 0.8, conv=3, chunk=32), 32), bare(attention(4, 2, 16, 16, 1.0, conv=4, rot=(4, 100.0)))])
    if which == "wide":     # sizes that the tensor-core kernels take (multiples of 16 and 64)
        return dict(base, vocab=200, width=128, logit_scale=0.8, token_side=dict(dim=32), layers=[
            moe(attention(4, 2, 64, 32, 0.12, conv=4, chunk=100, rot=(32, 5000.0)), 6, 2, 64, shared=64, groups=(3, 2), scale=1.5),
            dense(attention(8, 2, 32, 32, 0.2, conv=4, chunk=64, rot=(32, 1e4)), 192),
            moe(attention(8, 1, 48, 64, 0.15, conv=3, rot=(16, 1e4)), 4, 2, 64)])
    if which == "larger":   # widths, heads and experts that the tcgen05 products take in long portions
        return dict(base, vocab=1000, width=512, logit_scale=0.6, token_side=dict(dim=64), layers=[
            moe(attention(8, 2, 128, 128, 0.09, conv=4, chunk=300, rot=(64, 1e5)), 8, 2, 256, shared=256, groups=(4, 2), scale=2.0),
            dense(attention(16, 4, 64, 64, 0.12, conv=4, chunk=256, rot=(64, 1e4)), 1024),
            moe(attention(4, 1, 96, 256, 0.1, conv=4, rot=(96, 1e4)), 6, 2, 256, groups=(2, 1))])
    if which == "only_attention":
        return dict(base, vocab=97, width=40, layers=[bare(attention(4, 2, 16, 12, 0.3, conv=3, chunk=13, rot=(4, 100.0), v_mix=False))])
    if which == "only_mixing":      # three layers whose values are those of the first, with convolutions that hardly do anything
        return dict(base, vocab=97, width=40, layers=[bare(attention(2, 2, 8, 12, 0.3, conv=c, chunk=20)) for c in (2, 1, 4)])
    if which == "only_experts":     # the mixer is tiny, the feed-forward dominates
        return dict(base, vocab=97, width=40, layers=[moe(attention(1, 1, 4, 4, 0.5, conv=2, chunk=3), 8, 3, 24, shared=24, groups=(4, 2), scale=1.5),
                                                      moe(attention(1, 1, 4, 4, 0.5, conv=2), 6, 2, 12, groups=(2, 1))])
    if which == "only_side":        # the token inputs dominate
        return dict(base, vocab=97, width=40, token_side=dict(dim=24), layers=[bare(attention(1, 1, 4, 4, 0.5, conv=2, chunk=3)) for _ in range(3)])
    raise KeyError(which)


PAGE_SIZE = {"larger": 16, "wide": 16, "mix": 16, "odd": 2, "one": 4, "sharp": 16, "only_attention": 4, "only_mixing": 8, "only_experts": 16,
             "only_side": 16}


def make_weights(cfg: dict, seed: int) -> dict:
    """name -> float32 tensor whose values are all representable in bfloat16."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]

    def mat(out, inp, gain=1.0):
        return torch.randn(out, inp, generator=g) * (gain / math.sqrt(inp))

    def uni(shape, a, b):
        return a + (b - a) * torch.rand(shape, generator=g)

    W = {"embed": torch.randn(cfg["vocab"], d, generator=g), "head": mat(cfg["vocab"], d, 2.0), "final.norm": uni((d,), 0.8, 1.2)}
    n = (cfg.get("token_side") or {}).get("dim")
    if n:
        W["side.embed"] = torch.randn(cfg["vocab"], n * len(cfg["layers"]), generator=g)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        W[p + "norm1"] = uni((d,), 0.8, 1.2)
        for name, c in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            W[q + name] = mat(c, d, 1.5)
            if m.get("conv"):
                W[q + name + ".conv"] = uni((c, m["conv"]), -0.8, 0.8)
        W[q + "q.norm"], W[q + "k.norm"] = uni((dk,), 0.7, 1.5), uni((dk,), 0.7, 1.5)
        W[q + "sink"], W[q + "g"], W[q + "o"] = uni((H,), -1.0, 3.0), mat(H, d, 1.5), mat(d, H * dv, 2.0)
        if m.get("v_mix"):
            W[q + "vmix"] = uni((), 0.2, 0.8)
        if n:
            W[p + "side.gate"], W[p + "side.proj"], W[p + "side.norm"] = mat(n, d, 1.5), mat(d, n, 1.0), uni((d,), 0.3, 0.9)
        mlp = L.get("mlp")
        if not mlp:
            continue
        W[p + "norm2"] = uni((d,), 0.8, 1.2)

        def glu(pre, ff):
            W[pre + "gate"], W[pre + "up"], W[pre + "down"] = mat(ff, d, 1.5), mat(ff, d, 1.5), mat(d, ff)
        if mlp["kind"] == "dense":
            glu(p + "mlp.", mlp["ff"])
            continue
        W[p + "mlp.router"] = mat(mlp["router"]["experts"], d, 2.0)
        for e in range(mlp["router"]["experts"]):
            glu(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            glu(p + "mlp.shared.", mlp["shared"]["ff"])
            W[p + "mlp.shared.sg"] = mat(1, d, 1.5)
    return {k: v.to(torch.bfloat16).float() for k, v in W.items()}


def build(which: str, seed: int):
    """(config.json's dict, weights) of a named test model."""
    cfg = config(which)
    return cfg, make_weights(cfg, seed)

"""A plain, slow implementation of the Burolorn design in float64, one function per mechanism.

It shares no code with the engine: whole sequences at once, no cache, no pages, dense score matrices, convolutions over padded
sequences.  ``forward`` takes the dict of config.json, a dict name -> tensor and the token ids of one sequence, and returns
the logits of every position and the residual stream after every layer.

Notation: T tokens, d width, H query heads, G key-value heads, E experts, n the size of a layer's token input.
"""
from __future__ import annotations

import math

import torch

F = torch.float64

# With ``rounding("bfloat16")`` active every product's result and every activation between products is
# rounded to bfloat16 once, as a 16-bit engine does; what the design keeps in 32 bit is not.
_round = [lambda x: x]


class rounding:
    def __init__(self, kind):
        self.fn = (lambda x: x.to(torch.bfloat16).to(F)) if kind == "bfloat16" else (lambda x: x)

    def __enter__(self):
        self.old = _round[0]
        _round[0] = self.fn

    def __exit__(self, *a):
        _round[0] = self.old


def rnd(x):
    return _round[0](x)


def lin(h, w):
    return rnd(h @ w.to(F).T)


# ---------------------------------------------------------------- norms and activations

def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w.to(F)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def glu(h, W, p):
    """A gated feed-forward: down(silu(gate h) * up h)."""
    return lin(rnd(silu(lin(h, W[p + "gate"])) * lin(h, W[p + "up"])), W[p + "down"])


# ---------------------------------------------------------------- the mixer

def causal_conv(u, w):
    """u [T, C], w [C, taps]: the last tap meets the current token, zeros stand before the first one; no activation."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=F), u])
    return sum(padded[j:j + u.shape[0]] * w[:, j].to(F) for j in range(taps))


def rotate_halves(x, pos, rot):
    """x [T, heads, n]: entries i and i + dims/2 of the first rot.dims are turned together by pos * base^(-2i/dims); the rest pass."""
    dims = int(rot["dims"])
    half = dims // 2
    f = float(rot["base"]) ** (-2.0 * torch.arange(half, dtype=F) / dims)
    ang = (pos.to(F)[:, None] * f[None, :])[:, None, :]
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def chunk_mask(T, size):
    """[T, T]: query i (rows) sees key j <= i of its own chunk of ``size`` positions (None: every earlier key)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i // size == j // size if size is not None else j <= i)


def softmax_with_sink(scores, visible, sink):
    """scores [H, T, T]; ``sink`` [H]: one more term exp(sink_h) in every denominator, with no value."""
    s = scores.masked_fill(~visible, -math.inf)
    base = sink.to(F)[:, None, None]
    m = torch.maximum(s.max(-1, keepdim=True).values, base)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(base - m))


def mixed_values(v, first, lam):
    """The values of a later layer of the group: (1 - lam) v + lam first."""
    return (1.0 - lam) * v + lam * first


def attention(h, W, p, m, eps, first_values):
    """(output [T, d], this layer's values before mixing).  ``first_values``: the group's first layer's values, or None when the
    layer mixes nothing."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (lin(h, W[p + n]) for n in "qkv")
    if m.get("conv"):
        q, k, v = (rnd(causal_conv(u, W[p + n + ".conv"])) for n, u in zip("qkv", (q, k, v)))
    q = rms_norm(q.view(T, H, dk), W[p + "q.norm"], eps)
    k = rms_norm(k.view(T, G, dk), W[p + "k.norm"], eps)
    pos = torch.arange(T)
    if m.get("rot") and m["rot"]["dims"]:
        q, k = rotate_halves(q, pos, m["rot"]), rotate_halves(k, pos, m["rot"])
    q, k = rnd(q), rnd(k)
    own = v
    if first_values is not None:
        v = rnd(mixed_values(v, first_values, W[p + "vmix"].to(F)))
    kk = k.repeat_interleave(H // G, dim=1)
    vv = v.view(T, G, dv).repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * float(m["scale"])
    w = softmax_with_sink(s, chunk_mask(T, (m.get("mask") or {}).get("size"))[None], W[p + "sink"])
    y = torch.einsum("hij,jhd->ihd", w, vv)
    y = rnd(y * torch.sigmoid(lin(h, W[p + "g"]))[:, :, None])
    return lin(y.reshape(T, H * dv), W[p + "o"]), own


# ---------------------------------------------------------------- the feed-forward

MARGINS = None      # a list: every call of ``route`` appends its tokens' margins [T] here


def route(h, router_w, r):
    """(chosen [T, top], weights [T, top]): sigmoid scores; whole groups of neighbours drop out when the sum of their two largest
    scores is not among the ``keep`` best; the chosen scores divided by their sum, times the scale."""
    top, n = r["top"], router_w.shape[0]
    s = torch.sigmoid(h @ router_w.to(F).T)
    pick = s
    margin = torch.full((h.shape[0],), 9.0, dtype=F)
    groups = r.get("groups")
    if groups:
        per = n // groups["count"]
        score = torch.sort(s.view(-1, groups["count"], per), dim=-1, descending=True).values[..., :2].sum(-1)
        order = torch.sort(score, dim=-1, descending=True, stable=True)
        if groups["keep"] < groups["count"]:
            margin = torch.minimum(margin, order.values[:, groups["keep"] - 1] - order.values[:, groups["keep"]])
        kept = torch.zeros_like(score, dtype=torch.bool).scatter_(1, order.indices[:, :groups["keep"]], True)
        pick = pick.masked_fill(~kept.repeat_interleave(per, dim=1), -math.inf)
    ranked = torch.sort(pick, dim=-1, descending=True, stable=True)
    if top < n:
        margin = torch.minimum(margin, ranked.values[:, top - 1] - ranked.values[:, top])
    if MARGINS is not None:      # how far the last chosen is ahead of the first left out, and the last kept group of the next one
        MARGINS.append(margin)
    chosen = ranked.indices[:, :top]
    w = torch.gather(s, 1, chosen)
    return chosen, w / (w.sum(-1, keepdim=True) + 1e-20) * float(r["scale"] if r.get("scale") is not None else 1.0)


def experts(h, W, p, mlp):
    r = mlp["router"]
    chosen, weight = route(h, W[p + "router"], r)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        at = (chosen == e).nonzero()
        if at.numel():
            t, j = at[:, 0], at[:, 1]
            out[t] += weight[t, j][:, None] * glu(h[t], W, f"{p}e{e}.")
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ W[p + "shared.sg"].to(F).T) * glu(h, W, p + "shared.")
    return rnd(out)


# ---------------------------------------------------------------- the token input of a layer

def token_input(x, tokens, W, layer, n, eps):
    """What a layer adds to the stream for the tokens themselves: its part of the side table, gated by the stream."""
    p = f"l{layer}.side."
    e = W["side.embed"].to(F)[tokens][:, layer * n:(layer + 1) * n]
    g = rnd(gelu_tanh(rnd(x) @ W[p + "gate"].to(F).T) * e)
    return rms_norm(g @ W[p + "proj"].to(F).T, W[p + "norm"], eps)


# ---------------------------------------------------------------- the model

def forward(cfg: dict, W: dict, tokens):
    """(logits [T, vocab], stream after every layer [layers, T, d]), both float64."""
    eps = float(cfg["norm"]["eps"])
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"].to(F)[tokens]
    after, first_values = [], None
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        mixes = bool(m.get("v_mix"))
        y, own = attention(rnd(rms_norm(x, W[p + "norm1"], eps)), W, p + "mix.", m, eps, first_values if mixes else None)
        if mixes and first_values is None:
            first_values = own
        x = x + y
        if L.get("mlp"):
            h = rnd(rms_norm(x, W[p + "norm2"], eps))
            x = x + (glu(h, W, p + "mlp.") if L["mlp"]["kind"] == "dense" else experts(h, W, p + "mlp.", L["mlp"]))
        if cfg.get("token_side"):
            x = x + token_input(x, tokens, W, i, int(cfg["token_side"]["dim"]), eps)
        after.append(x.clone())
    h = rnd(rms_norm(x, W["final.norm"], eps))
    return (h @ W["head"].to(F).T) * float(cfg.get("logit_scale", 1.0)), torch.stack(after)

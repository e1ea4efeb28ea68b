"""A plain, slow implementation of the Vazunex design in float64, one function per mechanism.

It shares no code with the engine: whole sequences at once, no cache, no pages, token-by-token recurrences, dense score
matrices.  ``forward`` takes the dict of config.json, a dict name -> tensor and the token ids of one sequence, and returns
the logits of every position and the residual stream after every layer.

Notation: T tokens, d width, H heads, G key-value heads or groups, N state size, R latent size, E experts.
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

def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """The model's norm: the stored weight is the deviation from one."""
    return unit_rms(x, eps) * (1.0 + w.to(F))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def causal_conv(x, w, b=None):
    """x [T, C], w [C, taps]: the last tap meets the current token, zeros before the first one."""
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F), x])
    y = sum(padded[j:j + x.shape[0]] * w[:, j].to(F) for j in range(taps))
    return y if b is None else y + b.to(F)


# ---------------------------------------------------------------- mixers

def delta_recurrence(q, k, v, beta, g):
    """q, k [T, H, dk], v [T, H, dv], beta [T, H], g [T, H, dk]: per head S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=F)
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out)


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_delta(h, W, p, m, eps):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (rnd(silu(causal_conv(lin(h, W[p + n]), W[p + n + ".conv"]))) for n in "qkv")
    q = (unit_vector(q.view(T, G, dk)) / math.sqrt(dk)).repeat_interleave(H // G, dim=1)
    k = unit_vector(k.view(T, G, dk)).repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(lin(h, W[p + "b"]))
    a = lin(lin(h, W[p + "a1"]), W[p + "a2"]) + W[p + "dt_bias"].to(F)
    g = torch.exp(-torch.exp(W[p + "A_log"].to(F))[None, :, None] * softplus(a).view(T, H, dk))
    o = delta_recurrence(q, k, v.view(T, H, dv), beta, g)
    gate = torch.sigmoid(lin(lin(h, W[p + "g1"]), W[p + "g2"])).view(T, H, dv)
    y = rnd(unit_rms(o, eps) * W[p + "norm"].to(F) * gate)
    return lin(y.reshape(T, H * dv), W[p + "o"])


def ssd_recurrence(x, B, C, dt, A, D):
    """x [T, H, P], B, C [T, H, N], dt [T, H]: S <- exp(-A dt) S + dt B x^T, y = S^T C + D x."""
    T, H, P = x.shape
    S = torch.zeros(H, B.shape[-1], P, dtype=F)
    out = []
    for t in range(T):
        S = torch.exp(-A * dt[t])[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, C[t]) + D[:, None] * x[t])
    return torch.stack(out)


def mamba2(h, W, p, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(lin(h, W[p + "in"]), [inner, inner + 2 * G * N, H], dim=-1)
    xbc = rnd(silu(causal_conv(xbc, W[p + "conv"], W[p + "conv.b"])))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    B, C = (t.reshape(T, G, N).repeat_interleave(H // G, dim=1) for t in (B, C))
    dt = softplus(dt + W[p + "dt_bias"].to(F))
    y = ssd_recurrence(x.reshape(T, H, P), B, C, dt, torch.exp(W[p + "A_log"].to(F)), W[p + "D"].to(F))
    y = y.reshape(T, inner) * silu(z)
    y = rnd(unit_rms(y.view(T, m["norm_groups"], -1), eps).reshape(T, inner) * W[p + "norm"].to(F))
    return lin(y, W[p + "o"])


def rotate_halves(x, pos, rot):
    """x [T, ..., n]: entries i and i + dims/2 of the first rot.dims are turned together by pos * base^(-2i/dims); the rest pass."""
    dims = int(rot["dims"])
    half = dims // 2
    f = float(rot["base"]) ** (-2.0 * torch.arange(half, dtype=F) / dims)
    ang = (pos.to(F)[:, None] * f[None, :]).view([x.shape[0]] + [1] * (x.dim() - 2) + [half])
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def softmax_with_sink(scores, visible, sink):
    """scores [H, T, T]; ``sink`` [H]: one more term exp(sink_h) in every denominator, with no value."""
    s = scores.masked_fill(~visible, -math.inf)
    base = sink.to(F)[:, None, None]
    m = torch.maximum(s.max(-1, keepdim=True).values, base)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(base - m))


def window_mask(T, size):
    """[T, T]: query i (rows) sees key j with 0 <= i - j < size (``size`` None: every earlier key)."""
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (dist >= 0) & (dist < size if size is not None else dist >= 0)


def latent_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, dq, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = lin(h, W[p + "q"]).view(T, H, dq + dr)
    low = lin(h, W[p + "dkv"])
    c = rnd(unit_rms(low[:, :R], eps) * W[p + "dkv.norm"].to(F))
    q_plain, q_rot, shared = q[..., :dq], q[..., dq:], low[:, R:]
    if dr:
        q_rot, shared = rnd(rotate_halves(q_rot, pos, m["rot"])), rnd(rotate_halves(shared, pos, m["rot"]))
    k_plain = lin(c, W[p + "uk"]).view(T, H, dq)
    v = lin(c, W[p + "uv"]).view(T, H, dv)
    s = torch.einsum("ihd,jhd->hij", q_plain, k_plain)
    if dr:
        s = s + torch.einsum("ihd,jd->hij", q_rot, shared)
    s = s * float(m["scale"])
    w = softmax_with_sink(s, window_mask(T, (m.get("mask") or {}).get("size"))[None], W[p + "sink"])
    y = rnd(torch.einsum("hij,jhd->ihd", w, v)).reshape(T, H * dv)
    return lin(rnd(y * torch.sigmoid(lin(h, W[p + "g"]))), W[p + "o"])


# ---------------------------------------------------------------- the feed-forward

MARGINS = None      # a list: every call of ``route`` appends its tokens' margins [T] here


def route(h, router_w, correction, r):
    """(chosen [T, top], weights [T, top]): softmax over all outputs; the correction joins the choice only; whole groups of
    neighbours drop out when their best choice score is not among the ``keep`` best."""
    top, n = r["top"], router_w.shape[0]
    s = torch.softmax(h @ router_w.to(F).T, dim=-1)
    pick = s + correction.to(F)
    margin = torch.full((h.shape[0],), 9.0, dtype=F)
    groups = r.get("groups")
    if groups:
        per = n // groups["count"]
        best = pick.view(-1, groups["count"], per).max(-1).values
        order = torch.sort(best, dim=-1, descending=True, stable=True)
        if groups["keep"] < groups["count"]:
            margin = torch.minimum(margin, order.values[:, groups["keep"] - 1] - order.values[:, groups["keep"]])
        kept = torch.zeros_like(best, dtype=torch.bool).scatter_(1, order.indices[:, :groups["keep"]], True)
        pick = pick.masked_fill(~kept.repeat_interleave(per, dim=1), -math.inf)
    ranked = torch.sort(pick, dim=-1, descending=True, stable=True)
    if top < n:
        margin = torch.minimum(margin, ranked.values[:, top - 1] - ranked.values[:, top])
    if MARGINS is not None:      # how far the last chosen is ahead of the first left out, and the last kept group of the next one
        MARGINS.append(margin)
    chosen = ranked.indices[:, :top]
    return chosen, torch.gather(s, 1, chosen) * float(r.get("scale", 1.0))


def expert(h, W, p):
    return lin(rnd(silu(lin(h, W[p + "gate"])) * lin(h, W[p + "up"])), W[p + "down"])


def experts(h, W, p, mlp):
    r = mlp["router"]
    chosen, weight = route(h, W[p + "router"], W[p + "correction"], r)
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r.get("identity", 0)):
        at = (chosen == e).nonzero()
        if at.numel():
            t, j = at[:, 0], at[:, 1]
            y = expert(h[t], W, f"{p}e{e}.") if e < r["experts"] else h[t]      # the last outputs hand the input on
            out[t] += weight[t, j][:, None] * y
    return out


# ---------------------------------------------------------------- the model

MIXERS = {"channel_delta": channel_delta, "mamba2": mamba2, "latent_attention": latent_attention}


def forward(cfg: dict, W: dict, tokens):
    """(logits [T, vocab], stream after every layer [layers, T, d]), both float64."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x = offset_norm(W["embed"].to(F)[torch.as_tensor(tokens, dtype=torch.long)], W["embed.norm"], eps)
    after = []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + mult * MIXERS[L["type"]](rnd(offset_norm(x, W[p + "norm1"], eps)), W, p + "mix.", L["mixer"], eps)
        if L.get("mlp"):
            x = x + mult * experts(rnd(offset_norm(x, W[p + "norm2"], eps)), W, p + "mlp.", L["mlp"])
        after.append(x.clone())
    h = rnd(offset_norm(x, W["final.norm"], eps))
    return (h @ W["head"].to(F).T) * float(cfg.get("logit_scale", 1.0)), torch.stack(after)

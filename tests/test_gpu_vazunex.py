"""The Vazunex design in the engine against the plain float64 implementation, on the GPU, in 32 bit and in bfloat16:
each mechanism alone (one-mechanism models, single kernels, and the stream after every layer), each request whole,
prefill against token-by-token decoding, portions down to two tokens, mixed batches with pages and slots that are used
again, keys just inside and just outside a window and at page borders, states that carry something far back, long decoding,
and greedy generation through ``LMBackend``, the command line and the replay command."""
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import helpers
import plain_vazunex as plain
import vazunex_helpers as vh

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda:0"
# 32 bit: the largest difference of a logit (or a stream entry) as a fraction of the largest value of its request's
# reference.  bfloat16: the root mean square of a position's differences as a fraction of that of the request's
# reference logits, and at most three times what rounding alone causes.
TOL = {"float32": 2e-5, "bfloat16": 6e-2}
LENGTHS = {"wide": [250, 5, 199, 64], "mix": [3, 37, 60, 121], "odd": [1, 7, 26, 45], "one": [2, 25, 33, 58], "sharp": [1, 40, 97, 150],
           "only_delta": [1, 9, 40, 75], "only_ssd": [1, 2, 33, 70], "only_latent": [2, 30, 47], "only_experts": [1, 6, 21, 50]}
_cache = {}


def model(tmp_path_factory, which):
    if which not in _cache:
        cfg, W = vh.build(which, 31 + len(which))
        folder = vh.write_folder(tmp_path_factory.mktemp("vazunex"), which, cfg, W)
        _cache[which] = (cfg, W, folder)
    return _cache[which]


def make_runner(folder, which, dtype, num_pages=None, max_batch=4, max_seq_len=256, **kw):
    from delta_b200.config import EngineConfig
    from delta_b200.engine.step import ModelRunner
    ps = vh.PAGE_SIZE[which] if isinstance(which, str) else int(which)
    cfg = EngineConfig(max_batch=max_batch, max_seq_len=max_seq_len, page_size=ps, dtype=dtype,
                       num_pages=num_pages if num_pages is not None else max_batch * (max_seq_len // ps), **kw)
    return ModelRunner(folder, engine_config=cfg)


CLOSE_CALL = 0.01      # a router's choice decided by less than this (in choice scores) may fall either way once the input is rounded to bfloat16


class Noise(list):
    """Per request and position the error that bfloat16 rounding alone causes: the plain implementation with rounding against
    itself without, and at least twice the median of that over the positions.  ``margins``: per request and position the smallest
    margin by which any router decided (which group is kept, which output is chosen)."""
    margins = None


def routed(cfg, W, t):
    plain.MARGINS = []
    logits = plain.forward(cfg, W, t)[0]
    m = plain.MARGINS
    plain.MARGINS = None
    return logits, (torch.stack(m).min(dim=0).values if m else torch.full((len(t),), 9.0))


def rounding_noise(cfg, W, toks, refs):
    out = Noise()
    out.margins = []
    for t, ref in zip(toks, refs):
        _, margins = routed(cfg, W, t)
        with plain.rounding("bfloat16"):
            em, _ = routed(cfg, W, t)
        out.margins.append(margins)
        err = (em - ref).pow(2).mean(dim=1).sqrt()
        calm = err[margins >= CLOSE_CALL]
        out.append(torch.clamp(err, min=2.0 * (calm.median().item() if calm.numel() else err.median().item())))
    return out


def compare(results, refs, lengths, dtype, what, noise=None):
    worst = 0.0
    for i, n in enumerate(lengths):
        got = helpers.stack_positions(results, i, n).double()
        if dtype == "float32":
            err = (got - refs[i]).abs().max(dim=1).values
            scale = refs[i].abs().max().item()
        else:
            err = (got - refs[i]).pow(2).mean(dim=1).sqrt()
            scale = refs[i].pow(2).mean().sqrt().item()
        allowed = torch.full_like(err, TOL[dtype] * scale)
        if noise is not None:
            allowed = torch.maximum(allowed, 3.0 * noise[i % len(noise)])
        bad = (err > allowed).nonzero()[:, 0].tolist()
        if noise is not None:
            # bfloat16: a close call of a router ends the comparison of the request; otherwise one position in fifty may be over
            # the bound (an estimate from one rounded run), by less than three times.
            outliers = []
            for p in bad:
                if noise.margins[i % len(noise)][:p + 1].min() < CLOSE_CALL:
                    err, bad = err[:p], [q for q in bad if q < p]
                    break
                if err[p] <= 3.0 * allowed[p]:
                    outliers.append(p)
            if len(outliers) <= max(1, len(err) // 50):
                bad = [q for q in bad if q not in outliers]
            if not err.numel():
                continue
        if bad:
            p = bad[0]
            raise AssertionError(f"{what}: request {i} first differs at position {p} (of {n}): error {err[p].item():.3e}, "
                                 f"allowed {allowed[p].item():.3e}")
        worst = max(worst, err.max().item() / scale)
    return worst


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(LENGTHS))
def test_every_way_of_cutting(tmp_path_factory, which, dtype):
    cfg, W, folder = model(tmp_path_factory, which)
    lengths = LENGTHS[which]
    toks = [helpers.random_tokens(n, cfg["vocab"], 200 + i) for i, n in enumerate(lengths)]
    refs = [plain.forward(cfg, W, t)[0] for t in toks]
    ps = vh.PAGE_SIZE[which]
    runner = make_runner(folder, which, dtype)
    noise = rounding_noise(cfg, W, toks, refs) if dtype == "bfloat16" else None
    worst = {}
    worst["whole"] = compare(helpers.run_schedule(runner, toks, helpers.whole(lengths)), refs, lengths, dtype, "whole", noise)
    worst["one by one"] = compare(helpers.run_schedule(runner, toks, helpers.last_one_by_one(lengths)), refs, lengths, dtype,
                                  "last 32 one by one", noise)
    for seed, sizes in ((1, (7, 2, 13, 2, 5, 3, 16, 2, 9)), (2, (2, 2, 3, 31, 2, 17, 33, 40))):
        res = helpers.run_schedule(runner, toks, helpers.changing_portions(lengths, seed=seed, sizes=sizes))
        worst[f"portions {seed}"] = compare(res, refs, lengths, dtype, "changing portions", noise)
    # mixed: more requests than slots, and a pool so small that pages of finished requests are used again
    prompt_lens = [max(1, n // 2) for n in lengths]
    steps, ends = helpers.mixed(lengths * 3, prompt_lens * 3, seed=3, max_live=3)
    tight = make_runner(folder, which, dtype, num_pages=helpers.peak_pages(steps, ends, ps), max_batch=3)
    res = helpers.run_schedule(tight, toks * 3, steps, ends)
    worst["mixed"] = compare(res, refs * 3, lengths * 3, dtype, "mixed with pages and slots used again", noise)
    print(f"\nworst logit error {which} {dtype}: " + ", ".join(f"{k} {v:.2e}" for k, v in worst.items()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_larger_sizes(tmp_path_factory, dtype):
    """Width 512, 8 experts, heads of 64 and 128: a 700-token prompt whole (well over a hundred rows an expert: the tcgen05 products; the
    warp-MMA attention; the recurrences in chunks), in portions of 256 beside a second request, and its last tokens one by one."""
    cfg, W, folder = model(tmp_path_factory, "larger")
    lengths = [700, 130]
    toks = [helpers.random_tokens(n, cfg["vocab"], 900 + i) for i, n in enumerate(lengths)]
    refs = [plain.forward(cfg, W, t)[0] for t in toks]
    noise = rounding_noise(cfg, W, toks, refs) if dtype == "bfloat16" else None
    runner = make_runner(folder, "larger", dtype, max_batch=2, max_seq_len=704, max_tokens_per_step=1024)
    compare(helpers.run_schedule(runner, toks, helpers.whole(lengths)), refs, lengths, dtype, "whole", noise)
    steps = [[(0, 0, 256), (1, 0, 100)], [(0, 256, 256), (1, 100, 1)], [(0, 512, 180), (1, 101, 29)]] + [[(0, p, 1)] for p in range(692, 700)]
    compare(helpers.run_schedule(runner, toks, steps), refs, lengths, dtype, "portions of 256 beside a second request", noise)


@pytest.mark.parametrize("which", ["mix", "odd", "one", "sharp", "only_delta", "only_ssd", "only_latent", "only_experts"])
def test_stream_after_every_layer(tmp_path_factory, which):
    """32 bit: the residual stream after every layer, for a prompt in one step and for the same prompt cut in two (portions that run in
    chunks, and short ones whose tokens are taken in turn)."""
    from delta_b200.engine.step import RowInput
    cfg, W, folder = model(tmp_path_factory, which)
    toks = helpers.random_tokens(75, cfg["vocab"], 5)
    _, after = plain.forward(cfg, W, toks)
    runner = make_runner(folder, which, "float32")
    for cut in (75, 40, 11):
        slot = runner.cache.acquire_slot()
        got = []
        for a, b in ((0, cut), (cut, 75)):
            if a == b:
                continue
            runner.capture = {"layer_totals": []}
            runner.run_rows([RowInput(slot, toks[a:b], a, [])])
            got.append(torch.stack(runner.capture["layer_totals"]).cpu())
        runner.capture = None
        runner.cache.release_slot(slot)
        got = torch.cat(got, dim=1).double()
        assert got.shape == after.shape
        for r in range(after.shape[0]):
            err = (got[r] - after[r]).abs().max().item()
            assert err <= TOL["float32"] * after[r].abs().max().item(), f"{which}: layer {r} differs by {err:.3e} (cut at {cut})"


@pytest.mark.parametrize("which,dtype", [("mix", "float32"), ("odd", "float32"), ("mix", "bfloat16")])
def test_long_decoding(tmp_path_factory, which, dtype):
    """A short prompt, then 180 tokens one by one: pages fill one after the other and are given back behind the windows, which pass over
    decoded tokens only."""
    cfg, W, folder = model(tmp_path_factory, which)
    n = 185
    toks = [helpers.random_tokens(n, cfg["vocab"], 9)]
    refs = [plain.forward(cfg, W, toks[0])[0]]
    runner = make_runner(folder, which, dtype, max_batch=1)
    steps = [[(0, 0, 5)]] + [[(0, p, 1)] for p in range(5, n)]
    res = helpers.run_schedule(runner, toks, steps)
    noise = rounding_noise(cfg, W, toks, refs) if dtype == "bfloat16" else None
    print("\nlong decoding worst", compare(res, refs, [n], dtype, "long decoding", noise))
    assert all(g.pool.held_pages == 0 for g in runner.cache.groups.values())


def test_a_slot_used_again_starts_clean(tmp_path_factory):
    """Request B after request A in the same slot and pages equals B alone: the cache and the states of A are gone."""
    from delta_b200.engine.step import RowInput
    cfg, W, folder = model(tmp_path_factory, "mix")
    runner = make_runner(folder, "mix", "float32", max_batch=1, num_pages=8, max_seq_len=128)
    a, b = helpers.random_tokens(100, cfg["vocab"], 1), helpers.random_tokens(50, cfg["vocab"], 2)
    ref = plain.forward(cfg, W, b)[0]
    for toks in (a, b):
        slot = runner.cache.acquire_slot()
        assert slot == 0
        logits = runner.run_rows([RowInput(slot, toks, 0, list(range(len(toks))))])
        runner.cache.release_slot(slot)
    err = (logits.cpu().double() - ref).abs().max().item()
    assert err <= TOL["float32"] * ref.abs().max().item()


# ---- weights made so that one key decides ---------------------------------------------------------------------------

def crafted_needle(window, seed=77):
    """One latent-attention layer whose plain queries are minus its plain keys (W_q = -W_uk W_dkv, without the latent's norm weight), and
    token 1's embedding is minus token 0's: a query of token 1 meets a key of token 0 with the largest score there is, and no other
    key comes close.  Token 0 stands once, far back; token 1 is the last token: what the last position gives is the value of the far
    one while the window reaches it, and knows nothing of it when it does not."""
    full = dict(architecture="Vazunex", norm=dict(eps=1e-5), vocab=900, width=64, logit_scale=0.9, residual_mult=0.8, layers=[
        vh.bare(vh.latent(2, 16, 8, 16, 24, 0.25, window=window))])
    W = vh.make_weights(full, seed)
    dkv, uk = W["l0.mix.dkv"].double(), W["l0.mix.uk"].double()
    q = W["l0.mix.q"].view(2, 24, 64)
    for h in range(2):
        q[h, :16] = -(uk[16 * h:16 * h + 16] @ dkv[:24]).float().to(torch.bfloat16).float() * 0.5
        q[h, 16:] *= 0.1
    W["l0.mix.q"] = q.reshape(48, 64).to(torch.bfloat16).float()
    W["l0.mix.dkv.norm"] = torch.ones(24)
    W["embed"][1] = -W["embed"][0]
    W["l0.mix.sink"] = W["l0.mix.sink"] * 0.0 - 2.0
    return full, W


def needle_prompt(vocab, n, a_at, seed):
    g = torch.Generator().manual_seed(seed)
    toks = (torch.randperm(vocab - 2, generator=g)[:n] + 2).tolist()
    toks[a_at], toks[-1] = 0, 1
    return toks


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,distance", [(None, 17), (None, 561), (40, 39), (40, 40), (33, 32), (33, 33), (256, 255), (256, 256), (16, 15), (16, 16)])
def test_a_far_key_inside_and_outside_the_window(tmp_path_factory, dtype, window, distance):
    """The crafted key is read ``distance`` tokens later (at page borders, hundreds of tokens back, the last one inside a window and the
    first one outside): in a whole prompt, with the reader decoded alone, with the reader opening a portion, and with the key ending one."""
    cfg, W = crafted_needle(window)
    n = distance + 30
    a_at = n - 1 - distance
    toks = needle_prompt(cfg["vocab"], n, a_at, distance)
    ref = plain.forward(cfg, W, toks)[0]
    without = list(toks)
    without[a_at] = [t for t in range(2, cfg["vocab"]) if t not in toks][0]
    moved = (plain.forward(cfg, W, without)[0][-1] - ref[-1]).abs().max().item() / ref.abs().max().item()
    if window is None or distance < window:
        assert moved > 0.15, f"the crafted key does not carry the weight ({moved:.3f})"
    else:
        assert moved < 1e-9
    folder = vh.write_folder(tmp_path_factory.mktemp("needle"), f"needle{distance}", cfg, W)
    runner = make_runner(folder, 16, dtype, max_batch=2, max_seq_len=640, max_tokens_per_step=640)
    noise = rounding_noise(cfg, W, [toks], [ref]) if dtype == "bfloat16" else None
    b_at = n - 1
    for what, steps in (("whole", [[(0, 0, n)]]), ("the reader decoded alone", [[(0, 0, b_at - 3)]] + [[(0, p, 1)] for p in range(b_at - 3, n)]),
                        ("the reader opens a portion", [[(0, 0, 2)], [(0, 2, b_at - 4)], [(0, b_at - 2, 2)], [(0, b_at, 1)]]),
                        ("the key ends a portion", [[(0, 0, a_at + 1)], [(0, a_at + 1, n - a_at - 1)]])):
        compare(helpers.run_schedule(runner, [toks], steps), [ref], [n], dtype, what, noise)


def crafted_memory(kind, seed=5):
    """One recurrent layer whose state hardly decays: what token 0 wrote is still there hundreds of tokens later."""
    layer = vh.delta(2, 1, 16, 24, 3, 8, 8) if kind == "delta" else vh.ssd(2, 24, 16, 1, 3, 2)
    full = dict(architecture="Vazunex", norm=dict(eps=1e-5), vocab=900, width=64, logit_scale=0.9, layers=[vh.bare(layer)])
    W = vh.make_weights(full, seed)
    W["l0.mix.A_log"] = torch.full((2,), -3.0)
    W["l0.mix.dt_bias"] = W["l0.mix.dt_bias"] * 0.0 - (8.0 if kind == "delta" else 1.0)
    return vh.strip(full), W


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["delta", "ssd"])
def test_a_state_is_carried_far(tmp_path_factory, kind, dtype):
    """A token near the start moves the last logits by far more than the tolerance; whole, across portions that end inside and at the
    edges of the kernels' chunks of 32 tokens, and through decoding."""
    cfg, W = crafted_memory(kind)
    n = 200
    toks = helpers.random_tokens(n, cfg["vocab"], 3)
    ref = plain.forward(cfg, W, toks)[0]
    other = list(toks)
    other[1] = (other[1] + 1) % cfg["vocab"]
    moved = (plain.forward(cfg, W, other)[0][-1] - ref[-1]).abs().max().item() / ref.abs().max().item()
    assert moved > 20 * TOL["float32"], moved
    folder = vh.write_folder(tmp_path_factory.mktemp("memory"), kind, vh.strip(cfg), W)
    runner = make_runner(folder, 16, dtype, max_batch=2, max_seq_len=256)
    noise = rounding_noise(cfg, W, [toks], [ref]) if dtype == "bfloat16" else None
    for what, cuts in (("whole", [n]), ("at the chunks' edges", [32, 64, 160, n]), ("inside the chunks", [33, 66, 130, 133, 199, n]),
                       ("one token first", [1, 34, 67, n]), ("one by one behind a portion", [40] + list(range(41, n + 1)))):
        steps = [[(0, a, b - a)] for a, b in zip([0] + cuts[:-1], cuts)]
        compare(helpers.run_schedule(runner, [toks], steps), [ref], [n], dtype, what, noise)


# ---- single kernels against their equations ---------------------------------------------------------------------

def step_rows(lens, slots):
    """The device tensors that describe a step of rows with these lengths in these slots."""
    i32 = torch.int32
    starts = [sum(lens[:r]) for r in range(len(lens))]
    return dict(row_slot=torch.tensor(slots, dtype=i32, device=DEV), row_q_start=torch.tensor(starts, dtype=i32, device=DEV),
                row_q_len=torch.tensor(lens, dtype=i32, device=DEV)), starts


def chunk_base(lens, chunk):
    counts = [-(-n // chunk) for n in lens]
    return torch.tensor([sum(counts[:r]) for r in range(len(lens))], dtype=torch.int32, device=DEV), sum(counts), max(counts)


def plain_delta_from(S, q, k, v, beta, g):
    out = []
    for t in range(q.shape[0]):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("decays", ["weak", "mixed", "strong"])
@pytest.mark.parametrize("H,G,dk,dv", [(2, 1, 16, 24), (3, 3, 10, 7), (2, 2, 128, 64), (2, 1, 70, 33), (1, 1, 200, 20), (1, 1, 330, 9)])
def test_delta_rule_kernels(dtype, decays, H, G, dk, dv):
    """Tokens in turn and chunks of 32 from a state that is there already, rows of unequal lengths in shuffled slots, decays from almost one
    to zero (also side by side in one channel), and the state that is left."""
    from delta_b200.kernels import ops
    g = torch.Generator().manual_seed(H * 100 + dk)
    lens, slots = [1, 33, 70, 32], [2, 0, 4, 1]
    T = sum(lens)
    qkv = torch.randn(T, 2 * G * dk + H * dv, generator=g).to(dtype)
    qkv[3, :dk] = 0.0                                        # a zero query stays zero: the guard
    b = (torch.randn(T, H + 3, generator=g) * 2).to(dtype)
    a = torch.randn(T, H * dk + 5, generator=g) * 2
    A_log, dt_bias = {"weak": (torch.full((H,), -4.0), -4.0), "mixed": (torch.linspace(-2, 2, H), -1.0), "strong": (torch.full((H,), 3.0), 2.0)}[decays]
    dt_bias = torch.full((H * dk,), dt_bias)
    if decays == "mixed":
        a[::7] += 40.0                                       # single tokens forget everything
    state = torch.randn(5, H, dv, dk, generator=g)
    rows, starts = step_rows(lens, slots)
    scale, guard = 0.37, 1e-6
    x = qkv.double()
    unit = lambda t: t / torch.sqrt((t * t).sum(-1, keepdim=True) + guard)      # noqa: E731
    q = (unit(x[:, :G * dk].view(T, G, dk)) * scale).repeat_interleave(H // G, dim=1)
    k = unit(x[:, G * dk:2 * G * dk].view(T, G, dk)).repeat_interleave(H // G, dim=1)
    v = x[:, 2 * G * dk:].view(T, H, dv)
    dec = torch.exp(-torch.exp(A_log.double())[None, :, None] * plain.softplus(a[:, :H * dk].double() + dt_bias.double()).view(T, H, dk))
    on = dict(qkv=qkv.to(DEV), b=b.to(DEV), a=a.to(DEV), A_log=A_log.to(DEV), dt_bias=dt_bias.to(DEV))
    for chunked in (False, True):
        if chunked and not ops.delta_rule_chunked_supported(dk, dv):
            assert dk > 256
            continue
        st = state.to(DEV).clone()
        out = torch.full((T, H * dv), float("nan"), device=DEV)
        args = (on["qkv"], G * dk, 2 * G * dk, on["b"].data_ptr(), H + 3, on["a"], on["A_log"], on["dt_bias"], st, out)
        sizes = dict(H=H, G=G, dk=dk, dv=dv, q_scale=scale, guard=guard)
        if chunked:
            base, total, most = chunk_base(lens, ops.delta_rule_chunk())
            work = torch.full((total * H * ops.delta_rule_chunk_floats(dk, dv),), float("nan"), device=DEV)
            ops.delta_rule_chunked(*args, work, base, most, **sizes, **rows)
        else:
            ops.delta_rule(*args, **sizes, **rows)
        for r, n in enumerate(lens):
            s = slice(starts[r], starts[r] + n)
            o, S = plain_delta_from(state[slots[r]].double().transpose(1, 2), q[s], k[s], v[s], torch.sigmoid(b[s, :H].double()), dec[s])
            err = (out[s].cpu().double().view(n, H, dv) - o).abs().max().item() / o.abs().max().item()
            assert err < 1e-5, (chunked, r, err)
            err = (st[slots[r]].cpu().double().transpose(1, 2) - S).abs().max().item() / S.abs().max().item()
            assert err < 1e-5, (chunked, r, err)
        assert torch.equal(st[3].cpu(), state[3])            # a slot of no row
    # every row one token: the rows' lengths are not read
    n = len(lens)
    st = state.to(DEV).clone()
    out = torch.empty(T, H * dv, device=DEV)
    rows1, _ = step_rows([1] * n, slots)
    rows1["row_q_len"] = None
    ops.delta_rule(on["qkv"], G * dk, 2 * G * dk, on["b"].data_ptr(), H + 3, on["a"], on["A_log"], on["dt_bias"], st, out, **sizes, **rows1)
    for r in range(n):
        s = slice(r, r + 1)
        o, S = plain_delta_from(state[slots[r]].double().transpose(1, 2), q[s], k[s], v[s], torch.sigmoid(b[s, :H].double()), dec[s])
        assert (out[r].cpu().double().view(H, dv) - o[0]).abs().max().item() <= 1e-5 * o.abs().max().item()
        assert (st[slots[r]].cpu().double().transpose(1, 2) - S).abs().max().item() <= 1e-5 * S.abs().max().item()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("decays", ["weak", "mixed", "strong"])
@pytest.mark.parametrize("H,G,N,P", [(4, 2, 24, 16), (3, 1, 9, 14), (64, 2, 128, 64), (96, 4, 32, 40), (1, 1, 1, 1), (2, 2, 200, 33), (1, 1, 420, 5)])
def test_state_space_kernels(dtype, decays, H, G, N, P):
    """As for the delta rule: tokens in turn and chunks, narrow and wide slices of the channels, 16-byte copies and single loads."""
    from delta_b200.kernels import ops
    g = torch.Generator().manual_seed(H * 10 + N)
    lens, slots = [1, 33, 70, 32], [2, 0, 4, 1]
    T = sum(lens)
    ch = H * P + 2 * G * N
    xbc = torch.randn(T, ch, generator=g).to(dtype)
    dtraw = (torch.randn(T, H + 3, generator=g) * 2).to(dtype)
    A_log, bias = {"weak": (torch.full((H,), -4.0), -4.0), "mixed": (torch.linspace(-2, 2, H), -1.0), "strong": (torch.full((H,), 3.0), 2.0)}[decays]
    if decays == "mixed":
        dtraw[::7] += 30.0
    dt_bias, D = torch.full((H,), bias), torch.randn(H, generator=g)
    state = torch.randn(5, H, P, N, generator=g)
    rows, starts = step_rows(lens, slots)
    x = xbc[:, :H * P].double().view(T, H, P)
    B = xbc[:, H * P:H * P + G * N].double().view(T, G, N).repeat_interleave(H // G, dim=1)
    C = xbc[:, H * P + G * N:].double().view(T, G, N).repeat_interleave(H // G, dim=1)
    dt = plain.softplus(dtraw[:, :H].double() + bias)
    A = torch.exp(A_log.double())

    def reference(S, s):
        out = []
        for t in range(s.start, s.stop):
            S = torch.exp(-A * dt[t])[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
            out.append(torch.einsum("hnp,hn->hp", S, C[t]) + D.double()[:, None] * x[t])
        return torch.stack(out), S

    on = dict(xbc=xbc.to(DEV), dt=dtraw.to(DEV), A_log=A_log.to(DEV), dt_bias=dt_bias.to(DEV), D=D.to(DEV))
    for chunked in (False, True):
        if chunked and not ops.state_space_chunked_supported(N, P, dtype):
            assert N > 200
            continue
        st = state.to(DEV).clone()
        out = torch.full((T, H * P), float("nan"), device=DEV)
        args = (on["xbc"], on["dt"].data_ptr(), H + 3, on["A_log"], on["dt_bias"], on["D"], st, out)
        if chunked:
            base, total, most = chunk_base(lens, ops.state_space_chunk())
            work = torch.full((total * ops.state_space_chunk_floats(H, G),), float("nan"), device=DEV)
            ops.state_space_chunked(*args, work, base, total, most, H=H, G=G, N=N, P=P, **rows)
        else:
            ops.state_space(*args, H=H, G=G, N=N, P=P, **rows)
        for r, n in enumerate(lens):
            s = slice(starts[r], starts[r] + n)
            y, S = reference(state[slots[r]].double().transpose(1, 2), s)
            err = (out[s].cpu().double().view(n, H, P) - y).abs().max().item() / y.abs().max().item()
            assert err < 1e-5, (chunked, r, err)
            err = (st[slots[r]].cpu().double().transpose(1, 2) - S).abs().max().item() / S.abs().max().item()
            assert err < 1e-5, (chunked, r, err)
        assert torch.equal(st[3].cpu(), state[3])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps,C", [(2, 40), (3, 64), (4, 2048), (4, 42), (1, 24), (6, 48)])
def test_convolution_kernels(dtype, taps, C):
    """Rows of several tokens (the 16-byte kernel and the scalar one) and rows of one token each (convolution and state in one kernel): outputs
    and the inputs that are left, from a state that is there already."""
    from delta_b200.kernels import ops
    g = torch.Generator().manual_seed(taps * 1000 + C)
    for lens in ([1, 19, 2, 8], [1, 1, 1, 1]):
        slots, T = [3, 0, 4, 1], sum(lens)
        stride = C + (8 if C % 8 == 0 else 3)
        x = torch.randn(T, stride, generator=g).to(dtype)
        w, bias = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
        state = torch.randn(5, max(taps - 1, 1), C, generator=g)
        rows, starts = step_rows(lens, slots)
        tok_row = torch.tensor([r for r, n in enumerate(lens) for _ in range(n)], dtype=torch.int32, device=DEV)
        for b, silu, single in ((bias, True, False), (None, False, False), (bias, True, True)):
            if single and max(lens) > 1:
                continue
            st, out = state.to(DEV).clone(), torch.empty(T, C, dtype=dtype, device=DEV)
            ops.conv_silu(x.to(DEV), stride, w.to(DEV), b.to(DEV) if b is not None else None, st, out, tok_row=tok_row, silu=silu, single=single, **rows)
            for r, n in enumerate(lens):
                seq = torch.cat([state[slots[r]].double()[:taps - 1], x[starts[r]:starts[r] + n, :C].double()])
                want = sum(seq[j:j + n] * w[:, j].double() for j in range(taps)) + (b.double() if b is not None else 0.0)
                want = plain.silu(want) if silu else want
                tol = 1e-5 if dtype == torch.float32 else 1e-2
                assert (out[starts[r]:starts[r] + n].cpu().double() - want).abs().max().item() <= tol * max(1.0, want.abs().max().item())
                if taps > 1:
                    assert torch.equal(st[slots[r]].cpu(), seq[-(taps - 1):].float())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_small_kernels(dtype):
    """The normed embedding, the stream's step with a constant on the update, norms before and behind their gates with gates of either type."""
    from delta_b200.kernels import ops
    g = torch.Generator().manual_seed(2)
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    for d in (50, 1030):
        table, w = torch.randn(20, d, generator=g).to(dtype), torch.rand(d, generator=g) + 0.5
        toks = torch.tensor([3, 0, 19, 7], dtype=torch.int32)
        X = torch.empty(4, d, device=DEV)
        ops.embedding_pair(toks.to(DEV), table.to(DEV), X, norm_weight=w.to(DEV), eps=1e-4, kind="rms")
        want = plain.unit_rms(table[toks.long()].double(), 1e-4) * w.double()
        assert (X.cpu().double() - want).abs().max().item() <= 2e-6 * want.abs().max().item()
        y = torch.randn(4, d, generator=g).to(dtype)
        out = torch.empty(4, d, dtype=dtype, device=DEV)
        X0 = X.cpu().double()
        ops.residual_norm(X, out, updates=(y.to(DEV),), update_scale=0.3, weight=w.to(DEV), eps=1e-5, kind="rms")
        want = X0 + 0.3 * y.double()
        assert (X.cpu().double() - want).abs().max().item() <= 1e-6 * want.abs().max().item()
        want = plain.unit_rms(want, 1e-5) * w.double()
        assert (out.cpu().double() - want).abs().max().item() <= tol * want.abs().max().item()
    T, n = 5, 96
    o, w = torch.randn(T, n, generator=g), torch.rand(n, generator=g) + 0.5
    for gate_dtype in {dtype, torch.float32}:
        gate = torch.randn(T, n + 7, generator=g).to(gate_dtype)
        gd = gate.to(DEV)
        for group in (n, 24, 3):
            for first in (False, True):
                out = torch.empty(T, n, dtype=dtype, device=DEV)
                ops.gated_rms_norm(o.to(DEV), gd.data_ptr() + 7 * gd.element_size(), n + 7, w.to(DEV), out, 1e-5, group=group, gate_first=first, gate_dtype=gate_dtype)
                z = gate[:, 7:].double()
                x = o.double() * plain.silu(z) if first else o.double()
                want = plain.unit_rms(x.view(T, n // group, group), 1e-5).reshape(T, n) * w.double() * (1.0 if first else torch.sigmoid(z))
                assert (out.cpu().double() - want).abs().max().item() <= max(tol, 4e-6) * want.abs().max().item()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("outputs,top,groups,tokens", [(10, 2, (2, 1), 9), (9, 4, (3, 2), 40), (9, 1, (9, 4), 5), (24, 6, (4, 3), 2000), (7, 7, None, 3), (160, 8, (8, 3), 17),
                                                       (64, 2, (64, 2), 33), (12, 3, (1, 1), 8)])
def test_router_kernel(dtype, outputs, top, groups, tokens):
    """Softmax over all outputs, the correction in the choice only (choice scores below zero included), groups of neighbours, raw weights
    times a factor; tokens on several blocks."""
    from delta_b200.kernels import ops
    g = torch.Generator().manual_seed(outputs + top)
    d = 40
    x, w = torch.randn(tokens, d, generator=g).to(dtype), (torch.randn(outputs, d, generator=g) * 0.3).to(dtype)
    corr = torch.rand(outputs, generator=g) * 0.5 - 0.45
    z = torch.empty(tokens, outputs, device=DEV)
    choice, weight = torch.empty(tokens, top, dtype=torch.int32, device=DEV), torch.empty(tokens, top, device=DEV)
    ops.router(x.to(DEV), w.to(DEV), outputs, top, z, choice, weight, scoring="softmax_all", correction=corr.to(DEV), scale=1.7, normalize=False, groups=groups)
    r = dict(top=top, scale=1.7)
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    plain.MARGINS = []
    chosen, want = plain.route(x.double(), w, corr, r)
    sure = plain.MARGINS[0] > 1e-5
    plain.MARGINS = None
    assert sure.float().mean().item() > 0.9
    same = torch.sort(choice.cpu().long(), dim=-1), torch.sort(chosen, dim=-1)
    assert torch.equal(same[0].values[sure], same[1].values[sure])
    got = torch.gather(weight.cpu().double(), 1, same[0].indices)[sure]
    assert (got - torch.gather(want, 1, same[1].indices)[sure]).abs().max().item() <= 2e-6 * want.abs().max().item()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_experts_with_identities(dtype):
    """The whole feed-forward: tokens that choose only identities, only experts, and both; an expert nobody chooses."""
    from delta_b200.parts.experts import Experts
    g = torch.Generator().manual_seed(8)
    d, E, I, ff, top = 32, 4, 3, 24, 2
    W = {"x.router": torch.randn(E + I, d, generator=g), "x.correction": torch.zeros(E + I)}
    for e in range(E):
        W[f"x.e{e}.gate"], W[f"x.e{e}.up"], W[f"x.e{e}.down"] = (torch.randn(*s, generator=g) * 0.3 for s in ((ff, d), (ff, d), (d, ff)))
    W["x.correction"][1] = -3.0                              # never chosen
    W = {k: v.to(torch.bfloat16).float() for k, v in W.items()}
    part = Experts("x.", d, E, top, ff, limit=None, alpha=1.0, shift=0.0, scoring="softmax_all", correction=True, normalize=False, route_scale=1.5,
                   identity=I, wide_output=True)
    part.bind({k: v.to(dtype).to(DEV) if "correction" not in k else v.to(DEV) for k, v in W.items()})
    x = (torch.randn(70, d, generator=g) * 1.5).to(dtype)

    class Ctx:
        plain_kernels = frozenset()
        err = None
    out = part.forward(Ctx(), x.to(DEV)).cpu().double()
    mlp = dict(router=dict(experts=E, identity=I, top=top, scale=1.5))
    plain.MARGINS = []
    with plain.rounding("bfloat16" if dtype == torch.bfloat16 else None):
        want = plain.experts(x.double(), W, "x.", mlp)
    sure = plain.MARGINS[0] > 1e-4
    plain.MARGINS = None
    chosen, _ = plain.route(x.double(), W["x.router"], W["x.correction"], mlp["router"])
    kinds = (chosen >= E).sum(-1)
    assert set(kinds.tolist()) == {0, 1, 2} and not (chosen == 1).any()
    assert out.dtype == torch.float64 and (out - want)[sure].abs().max().item() <= (1e-5 if dtype == torch.float32 else 1e-2) * want.abs().max().item()


# ---- through the engine's own entry points -----------------------------------------------------------------------

def greedy_plain(cfg, W, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        logits, _ = plain.forward(cfg, W, toks)
        toks.append(int(torch.argmax(logits[-1])))
    return toks[len(prompt):]


@pytest.mark.parametrize("graph", [False, True])
def test_greedy_generation_through_the_backend(tmp_path_factory, graph):
    """``LMBackend``: more prompts than slots, a token budget that cuts prompts, decode steps (recorded or not)."""
    from delta_b200.engine import LMBackend
    cfg, W, folder = model(tmp_path_factory, "mix")
    prompts = [helpers.random_tokens(n, cfg["vocab"], 50 + n) for n in (4, 23, 9, 31, 2)]
    want = [greedy_plain(cfg, W, p, 10) for p in prompts]
    e = LMBackend(dtype="float32", device="cuda:0", cuda_graph_decode=graph)
    e.load_model(str(folder))
    e.setup_caches(max_batch_size=3, max_seq_length=64, page_size=16, max_tokens_per_step=16)
    got = e.generate(prompts, 10)
    assert got == want
    assert e.scheduler.stats["prefill_steps"] > 2
    if graph:
        assert e.runner.graph_replays > 0 and not e.runner.graph_fallbacks


def test_generation_survives_preemption(tmp_path_factory):
    """A pool too small for all running requests: the youngest is preempted and computed again from a fresh slot; the tokens are
    those of the plain implementation all the same."""
    from delta_b200.engine import LMBackend
    cfg, W, folder = model(tmp_path_factory, "mix")
    prompts = [helpers.random_tokens(n, cfg["vocab"], 80 + n) for n in (14, 15, 13)]
    want = [greedy_plain(cfg, W, p, 12) for p in prompts]
    e = LMBackend(dtype="float32", device="cuda:0")
    e.load_model(str(folder))
    e.setup_caches(max_batch_size=3, max_seq_length=32, page_size=4, max_tokens_per_step=16, num_pages=15)
    assert e.generate(prompts, 12) == want
    assert e.scheduler.stats["preemptions"] >= 1


def test_trace_replay_command(tmp_path_factory, tmp_path):
    """``bin/trace_run`` on a Vazunex folder: a prompt in portions beside another request's single tokens."""
    import numpy as np
    cfg, W, folder = model(tmp_path_factory, "odd")
    a, b = helpers.random_tokens(21, cfg["vocab"], 3), helpers.random_tokens(12, cfg["vocab"], 4)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:7], want=[6])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=a[7:9], want=[0, 1]), dict(id="b", tokens=b[:11], want=[10])], end=[]),
             dict(step=2, entries=[dict(id="b", tokens=b[11:], want=[0]), dict(id="a", tokens=a[9:], want=[11])], end=["a", "b"])]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128", "--page-size", "4"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    ra, rb = plain.forward(cfg, W, a)[0], plain.forward(cfg, W, b)[0]
    V = cfg["vocab"]
    got = {k: torch.from_numpy(np.fromfile(out / f"{k}.f32", dtype="<f4").reshape(-1, V)).double() for k in range(3)}
    want = {0: ra[[6]], 1: torch.cat([ra[[7, 8]], rb[[10]]]), 2: torch.cat([rb[[11]], ra[[20]]])}
    for k in range(3):
        assert got[k].shape == want[k].shape
        assert (got[k] - want[k]).abs().max().item() <= TOL["float32"] * want[k].abs().max().item()


def test_command_line_generates(tmp_path_factory, tmp_path):
    """``python -m delta_b200.cli`` on a Vazunex folder: the model class comes from config.json, prompts are scheduled and sampled."""
    import random
    from delta_b200 import cli
    cfg, W, folder = model(tmp_path_factory, "one")
    out = tmp_path / "result.json"
    rc = cli.main(["--model", str(folder), "--B", "3", "--max_len", "128", "--dataset", "random", "--prompt_len", "19", "--num_samples", "5",
                   "--max_new_tokens", "6", "--dtype", "float32", "--max_tokens_per_step", "32", "--out", str(out)])
    assert rc == 0
    res = json.loads(out.read_text())
    assert res["summary"]["requests"] == 5 and res["summary"]["generated_tokens"] == 30
    rng = random.Random(123)       # the command line's default seed draws the prompts
    prompt = [rng.randrange(cfg["vocab"]) for _ in range(19)]
    first = [r for r in res["results"] if r["request_id"] == 0][0]
    assert first["output_ids"] == greedy_plain(cfg, W, prompt, 6)

"""The Burolorn design in the engine against the plain float64 implementation, on the GPU, in 32 bit and in bfloat16:
each mechanism alone (one-mechanism models, single kernels, and the stream after every layer), each request whole,
prefill against token-by-token decoding, portions down to two tokens, mixed batches with pages and slots that are used
again, keys just inside and just outside a chunk and at page borders, long decoding, and greedy generation through
``LMBackend``, the command line and the replay command."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import burolorn_helpers as bh
import helpers
import plain_burolorn as plain

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda:0"
# 32 bit: the largest difference of a logit (or a stream entry) as a fraction of the largest value of its request's
# reference.  bfloat16: the root mean square of a position's differences as a fraction of that of the request's
# reference logits, and at most three times what rounding alone causes.
TOL = {"float32": 2e-5, "bfloat16": 6e-2}
LENGTHS = {"wide": [250, 5, 199, 64], "mix": [3, 37, 60, 121], "odd": [1, 7, 26, 45], "one": [2, 25, 33, 58], "sharp": [1, 40, 97, 150],
           "only_attention": [1, 9, 40, 75], "only_mixing": [1, 2, 33, 70], "only_experts": [1, 6, 21, 50], "only_side": [2, 30, 47]}
_cache = {}


def model(tmp_path_factory, which):
    if which not in _cache:
        cfg, W = bh.build(which, 31 + len(which))
        folder = bh.write_folder(tmp_path_factory.mktemp("burolorn"), which, cfg, W)
        _cache[which] = (cfg, W, folder)
    return _cache[which]


def make_runner(folder, which, dtype, num_pages=None, max_batch=4, max_seq_len=256, **kw):
    from delta_b200.config import EngineConfig
    from delta_b200.engine.step import ModelRunner
    ps = bh.PAGE_SIZE[which] if isinstance(which, str) else int(which)
    cfg = EngineConfig(max_batch=max_batch, max_seq_len=max_seq_len, page_size=ps, dtype=dtype,
                       num_pages=num_pages if num_pages is not None else max_batch * (max_seq_len // ps), **kw)
    return ModelRunner(folder, engine_config=cfg)


CLOSE_CALL = 0.02      # a router's choice decided by less than this (in scores, or in a group's sum of two) may fall either way once the input is
                       # rounded to bfloat16


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
    ps = bh.PAGE_SIZE[which]
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
    """Width 512, 8 experts, heads of 64 to 128 with values of 64 to 256: a 700-token prompt whole (well over a hundred rows an expert: the
    tcgen05 products; the warp-MMA attention over chunks that end inside its tiles), in portions of 256 beside a second request, and its
    last tokens one by one."""
    cfg, W, folder = model(tmp_path_factory, "larger")
    lengths = [700, 130]
    toks = [helpers.random_tokens(n, cfg["vocab"], 900 + i) for i, n in enumerate(lengths)]
    refs = [plain.forward(cfg, W, t)[0] for t in toks]
    noise = rounding_noise(cfg, W, toks, refs) if dtype == "bfloat16" else None
    runner = make_runner(folder, "larger", dtype, max_batch=2, max_seq_len=704, max_tokens_per_step=1024)
    compare(helpers.run_schedule(runner, toks, helpers.whole(lengths)), refs, lengths, dtype, "whole", noise)
    steps = [[(0, 0, 256), (1, 0, 100)], [(0, 256, 256), (1, 100, 1)], [(0, 512, 180), (1, 101, 29)]] + [[(0, p, 1)] for p in range(692, 700)]
    compare(helpers.run_schedule(runner, toks, steps), refs, lengths, dtype, "portions of 256 beside a second request", noise)


@pytest.mark.parametrize("which", ["mix", "odd", "one", "sharp", "only_attention", "only_mixing", "only_experts", "only_side"])
def test_stream_after_every_layer(tmp_path_factory, which):
    """32 bit: the residual stream after every layer, for a prompt in one step and for the same prompt cut in two (in the middle of pages,
    chunks and convolutions)."""
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
    """A short prompt, then 180 tokens one by one: pages fill one after the other and are given back behind the chunks, which pass over
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

def crafted_needle(chunk, seed=77):
    """One attention layer whose queries are minus its keys (W_q = -W_k, plain norm weights, convolutions that hand the current token on), and
    token 1's embedding is minus token 0's: a query of token 1 meets a key of token 0 with the largest score there is, and no other
    key comes close (few entries are rotated, so distance costs little).  Token 0 stands once, far back; token 1 is the last token: what the last
    position gives is the value of the far one while both stand in one chunk, and knows nothing of it when they do not."""
    cfg = dict(architecture="Burolorn", norm=dict(eps=1e-5), vocab=900, width=64, logit_scale=0.9, layers=[
        bh.bare(bh.attention(4, 2, 32, 16, 0.6, conv=4, chunk=chunk, rot=(2, 10000.0)))])
    W = bh.make_weights(cfg, seed)
    W["l0.mix.q"] = -W["l0.mix.k"].view(2, 1, 32, 64).expand(2, 2, 32, 64).reshape(128, 64).contiguous()
    for n in ("q", "k"):
        W[f"l0.mix.{n}.norm"] = torch.ones(32)
        W[f"l0.mix.{n}.conv"] = torch.zeros_like(W[f"l0.mix.{n}.conv"])
        W[f"l0.mix.{n}.conv"][:, -1] = 1.0
    W["embed"][1] = -W["embed"][0]
    return cfg, W


def needle_prompt(vocab, n, a_at, seed):
    g = torch.Generator().manual_seed(seed)
    toks = (torch.randperm(vocab - 2, generator=g)[:n] + 2).tolist()
    toks[a_at], toks[-1] = 0, 1
    return toks


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunk,key_at,reader_at", [
    (None, 3, 20), (None, 15, 576), (None, 16, 577),                       # every earlier key: across page borders, hundreds of tokens back
    (600, 0, 599), (600, 0, 600), (40, 40, 79), (40, 39, 79), (40, 40, 80), (40, 79, 80), (33, 33, 65), (33, 32, 65), (33, 32, 33),
    (256, 256, 511), (256, 255, 511), (16, 16, 31), (16, 15, 31), (16, 31, 32), (300, 301, 599), (300, 299, 300)])
def test_a_far_key_inside_and_outside_the_chunk(tmp_path_factory, dtype, chunk, key_at, reader_at):
    """The crafted key is the chunk's first token or the last one before it, the reader the chunk's last token or its first: in a whole prompt,
    with the reader decoded alone, with the reader opening a portion, with the key ending one, and with portions cut at the chunk's edge."""
    cfg, W = crafted_needle(chunk)
    n = reader_at + 1
    toks = needle_prompt(cfg["vocab"], n, key_at, reader_at)
    ref = plain.forward(cfg, W, toks)[0]
    without = list(toks)
    without[key_at] = [t for t in range(2, cfg["vocab"]) if t not in toks][0]
    W_v = dict(W)      # (the value's convolution would carry a near key's token along: it is left out of this check)
    W_v["l0.mix.v.conv"] = torch.zeros_like(W["l0.mix.v.conv"])
    W_v["l0.mix.v.conv"][:, -1] = 1.0
    a, b = plain.forward(cfg, W_v, toks)[0][-1], plain.forward(cfg, W_v, without)[0][-1]
    moved = (a - b).abs().max().item() / a.abs().max().item()
    if chunk is None or key_at // chunk == reader_at // chunk:
        assert moved > 0.1, f"the crafted key does not carry the weight ({moved:.3f})"
    else:
        assert moved < 1e-9
    folder = bh.write_folder(tmp_path_factory.mktemp("needle"), f"needle{key_at}_{reader_at}", cfg, W)
    runner = make_runner(folder, 16, dtype, max_batch=2, max_seq_len=640, max_tokens_per_step=640)
    noise = rounding_noise(cfg, W, [toks], [ref]) if dtype == "bfloat16" else None
    edge = chunk if chunk and chunk < reader_at else 7
    for what, cuts in (("whole", [n]), ("the reader decoded alone", [reader_at - 4, reader_at - 3, reader_at - 2, reader_at - 1, reader_at, n]),
                       ("the reader opens a portion", [2, max(3, reader_at - 2), reader_at, n]), ("the key ends a portion", [key_at + 1, n]),
                       ("cut at the chunk's edge", [edge, n]), ("cut behind the chunk's edge", [edge + 1, n]), ("cut before it", [edge - 1, n])):
        cuts = sorted({c for c in cuts if 0 < c <= n})
        steps = [[(0, a, b - a)] for a, b in zip([0] + cuts[:-1], cuts)]
        compare(helpers.run_schedule(runner, [toks], steps), [ref], [n], dtype, what, noise)


# ---- single kernels against their equations ---------------------------------------------------------------------

def step_rows(lens, slots, before):
    """The device tensors that describe a step of rows with these lengths in these slots."""
    i32 = dict(dtype=torch.int32, device=DEV)
    starts = [sum(lens[:r]) for r in range(len(lens))]
    rows = dict(row_slot=torch.tensor(slots, **i32), row_q_start=torch.tensor(starts, **i32), row_q_len=torch.tensor(lens, **i32))
    toks = dict(tok_pos=torch.tensor([b + i for b, n in zip(before, lens) for i in range(n)], **i32),
                tok_row=torch.tensor([r for r, n in enumerate(lens) for _ in range(n)], **i32))
    return rows, toks, starts


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps", [0, 1, 2, 3, 4, 6])
@pytest.mark.parametrize("H,KV,dk,dv,rot,interleaved", [(4, 2, 64, 32, 32, False), (3, 1, 128, 128, 128, False), (2, 2, 30, 66, 10, True),
                                                        (2, 1, 200, 24, 64, False), (3, 3, 11, 7, 4, False), (1, 1, 2, 2, 0, False),
                                                        (4, 2, 128, 64, 64, False), (2, 2, 64, 64, 8, False), (5, 1, 64, 128, 0, False)])
def test_convolution_norm_rotation_and_append(dtype, taps, H, KV, dk, dv, rot, interleaved):
    """From projected rows to queries and cache rows, with inputs of earlier steps in the state: the kernels that keep heads in registers and
    the one for any size, rows of several tokens and steps of single ones, value mixing of every kind, shuffled pages; and the state that
    is left."""
    for lens in ([1, 19, 2, 8], [1, 1, 1, 1]):
        check_conv_append(dtype, taps, H, KV, dk, dv, rot, interleaved, lens, [9, 0, 30, 5])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps,H,KV,dk,dv", [(4, 9, 3, 128, 64), (3, 8, 4, 64, 128), (2, 12, 2, 96, 32), (4, 8, 2, 64, 64), (4, 8, 2, 128, 128)])
def test_convolution_over_long_portions(dtype, taps, H, KV, dk, dv):
    """Enough tokens for the tiles of several tokens a warp, whose edges fall inside rows, between them and on rows of one or two tokens."""
    check_conv_append(dtype, taps, H, KV, dk, dv, 32, False, [3, 1001, 1, 2, 1500], [0, 57, 9, 0, 700], ps=16)


def check_conv_append(dtype, taps, H, KV, dk, dv, rot, interleaved, lens, before, ps=4):
    from delta_b200.kernels import ops
    g = torch.Generator().manual_seed(taps * 100 + dk)
    C = (H + KV) * dk + KV * dv
    tol = 3e-6 if dtype == torch.float32 else 1e-2
    slots, T = [3, 0, 4, 1, 5][:len(lens)], sum(lens)
    src = torch.randn(T, C + 8, generator=g).to(dtype)
    w = torch.randn(max(taps, 1), C, generator=g)
    state = torch.randn(7, max(taps - 1, 1), C, generator=g).to(dtype).float()      # (what a state holds are inputs as they were projected)
    qn, kn = torch.rand(dk, generator=g) + 0.5, torch.rand(dk, generator=g) + 0.5
    ang = torch.arange(max(b + n for b, n in zip(before, lens)), dtype=plain.F)[:, None] * 50.0 ** (-2.0 * torch.arange(max(rot // 2, 1), dtype=plain.F) / max(rot, 2))[None]
    table = torch.stack([torch.cos(ang), torch.sin(ang)], dim=-1).float()
    rows, toks, starts = step_rows(lens, slots, before)
    per = max(-(-(b + n) // ps) for b, n in zip(before, lens))
    n_pages = per * len(lens) + 3
    bt = torch.randperm(n_pages, generator=g)[:per * len(lens)].view(len(lens), per).int()
    first0 = torch.randn(T, KV * dv, generator=g).to(dtype)
    for mix in (None, "first", 0.3):
        for single in ((False, True) if max(lens) == 1 else (False,)):
            st, cache = state.to(DEV).clone(), torch.zeros(n_pages, KV, ps, dk + dv, dtype=dtype, device=DEV)
            q, first, err = torch.empty(T, H * dk, dtype=dtype, device=DEV), first0.to(DEV).clone(), ops.new_error_record(DEV)
            dev = dict(src=src.to(DEV), w=w.to(DEV), bt=bt.to(DEV), qn=qn.to(DEV), kn=kn.to(DEV), table=table.to(DEV))
            ops.rows_conv_append(dev["src"], q, dev["w"] if taps else None, st if taps > 1 else None, toks["tok_pos"], toks["tok_row"], dev["bt"], cache,
                                 H=H, KV=KV, dk=dk, dv=dv, ps=ps, row_width=dk + dv, k_off=0, v_off=dk, table=dev["table"] if rot else None,
                                 rot_dims=rot, interleaved=interleaved, q_norm=dev["qn"], k_norm=dev["kn"], eps=1e-5, first=first, mix=mix,
                                 single=single, err=err, **rows)
            ops.raise_if_error(err)
            q, cache, first, st = q.cpu().double(), cache.cpu().double(), first.cpu().double(), st.cpu()
            for r, n in enumerate(lens):
                x = src[starts[r]:starts[r] + n, :C].double()
                seq = torch.cat([state[slots[r]].double()[:max(taps - 1, 0)], x])
                u = sum(seq[j:j + n] * w[j].double() for j in range(taps)) if taps else x
                pos = torch.arange(before[r], before[r] + n)
                heads = []
                for part, weight in ((u[:, :H * dk].view(n, H, dk), qn), (u[:, H * dk:(H + KV) * dk].view(n, KV, dk), kn)):
                    y = plain.rms_norm(part, weight, 1e-5)
                    if rot:
                        perm = [2 * i for i in range(rot // 2)] + [2 * i + 1 for i in range(rot // 2)] if interleaved else list(range(rot))
                        y = y.clone()
                        y[..., perm] = plain.rotate_halves(y[..., perm], pos, dict(base=50.0, dims=rot))
                    heads.append(y)
                v = u[:, (H + KV) * dk:]
                f = first0[starts[r]:starts[r] + n].double()
                if mix == "first":
                    assert (first[starts[r]:starts[r] + n] - v).abs().max().item() <= tol * v.abs().max().item()
                if isinstance(mix, float):
                    v = plain.mixed_values(v, f, mix)
                    assert torch.equal(first[starts[r]:starts[r] + n], f)
                got = cache[bt[r].long()[pos // ps], :, pos % ps]      # [n, KV, dk + dv]
                for a, b in ((q[starts[r]:starts[r] + n].view(n, H, dk), heads[0]), (got[..., :dk], heads[1]), (got[..., dk:], v.reshape(n, KV, dv))):
                    assert (a - b).abs().max().item() <= tol * max(1.0, b.abs().max().item()), (r, mix, single)
                if taps > 1:
                    assert torch.equal(st[slots[r]], seq[-(taps - 1):].float())
            if taps > 1:
                assert torch.equal(st[2], state[2])            # a slot of no row


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_stream_step_with_a_normed_update(dtype):
    """x <- x + (y1 + y2) + rms(y3) w3, then the norm of it: the form that keeps the row in registers (up to two groups a thread), the one for
    any width, chosen rows without writing back, and the plain rounded stream."""
    from delta_b200.kernels import ops
    g = torch.Generator().manual_seed(4)
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    for d in (50, 64, 1032, 8192, 9216):
        x0, w, w3 = torch.randn(5, d, generator=g), torch.rand(d, generator=g) + 0.5, torch.rand(d, generator=g) + 0.5
        y1, y2, y3 = (torch.randn(5, d, generator=g).to(dtype) for _ in range(3))
        extra, vec, b = torch.randn(5, d, generator=g), torch.randn(d, generator=g), torch.randn(d, generator=g)
        on = {k: v.to(DEV) for k, v in dict(w=w, w3=w3, y1=y1, y2=y2, y3=y3, extra=extra, vec=vec, b=b).items()}
        n3 = plain.rms_norm(y3.double(), w3, 1e-3)
        for updates, normed, ex, vc in (((), True, False, False), (("y1",), True, False, False), (("y1", "y2"), False, True, True), (("y1", "y2"), True, True, True)):
            want = x0.double() + 0.7 * sum((on[k].cpu().double() for k in updates), torch.zeros(5, d, dtype=plain.F))
            want = want + (n3 if normed else 0.0) + (extra.double() if ex else 0.0) + (vec.double() if vc else 0.0)
            kw = dict(updates=tuple(on[k] for k in updates), update_scale=0.7, normed=(on["y3"], on["w3"], 1e-3) if normed else None,
                      extra=on["extra"] if ex else None, vec=on["vec"] if vc else None)
            for kind in ("rms", "layer"):
                c = want - want.mean(-1, keepdim=True) if kind == "layer" else want
                normal = plain.rms_norm(c, w, 1e-5) + b.double()
                X, out = x0.to(DEV), torch.empty(5, d, dtype=dtype, device=DEV)
                ops.residual_norm(X, out, weight=on["w"], bias=on["b"], eps=1e-5, kind=kind, **kw)
                assert (X.cpu().double() - want).abs().max().item() <= 1e-6 * want.abs().max().item()
                assert (out.cpu().double() - normal).abs().max().item() <= tol * normal.abs().max().item()
                rows = torch.tensor([3, 0], dtype=torch.int32, device=DEV)
                X, out = x0.to(DEV), torch.empty(2, d, dtype=dtype, device=DEV)
                ops.residual_norm(X, out, weight=on["w"], bias=on["b"], eps=1e-5, kind=kind, rows=rows, write_back=False, **kw)
                assert torch.equal(X.cpu(), x0) and (out.cpu().double() - normal[[3, 0]]).abs().max().item() <= tol * normal.abs().max().item()
            X, out = x0.to(DEV), torch.empty(5, d, dtype=dtype, device=DEV)
            ops.residual_norm(X, out, **kw)
            assert (out.cpu().double() - want).abs().max().item() <= tol * want.abs().max().item()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,parts,index", [(7, 3, 1), (24, 2, 0), (24, 2, 1), (300, 1, 0)])
def test_table_gate(dtype, n, parts, index):
    from delta_b200.kernels import ops
    from delta_b200.parts.feed_forward import GELU_TANH_GATE
    g = torch.Generator().manual_seed(n)
    z, table = (torch.randn(9, n, generator=g) * 2).to(dtype), torch.randn(13, parts * n, generator=g).to(dtype)
    toks = torch.tensor([0, 12, 5, 5, 3, 1, 7, 11, 2], dtype=torch.int32)
    err = ops.new_error_record(DEV)
    out = ops.table_gate(z.to(DEV), toks.to(DEV), table.to(DEV), index * n, torch.empty(9, n, dtype=dtype, device=DEV), GELU_TANH_GATE["alpha"],
                         GELU_TANH_GATE["cubic"], err=err)
    ops.raise_if_error(err)
    want = plain.gelu_tanh(z.double()) * table.double()[toks.long(), index * n:(index + 1) * n]
    assert (out.cpu().double() - want).abs().max().item() <= (2e-6 if dtype == torch.float32 else 1e-2) * want.abs().max().item()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("experts,top,groups,tokens", [(8, 2, (2, 1), 9), (9, 4, (3, 2), 40), (9, 1, (9, 4), 5), (24, 6, (4, 3), 2000), (7, 7, None, 3),
                                                       (160, 8, (8, 3), 17), (64, 2, (64, 2), 33), (12, 3, (1, 1), 8), (12, 2, (6, 3), 300)])
def test_router_kernel(dtype, experts, top, groups, tokens):
    """Sigmoid scores, groups ranked by the sum of their two largest (of their only one in groups of one), weights divided by their sum, times
    a factor; tokens on several blocks; another column (a shared expert's gate) behind the experts'."""
    from delta_b200.kernels import ops
    g = torch.Generator().manual_seed(experts + top)
    d = 40
    x, w = torch.randn(tokens, d, generator=g).to(dtype), (torch.randn(experts + 1, d, generator=g) * 0.3).to(dtype)
    z = torch.empty(tokens, experts + 1, device=DEV)
    choice, weight = torch.empty(tokens, top, dtype=torch.int32, device=DEV), torch.empty(tokens, top, device=DEV)
    ops.router(x.to(DEV), w.to(DEV), experts, top, z, choice, weight, scoring="sigmoid", scale=1.7, groups=groups, group_score="top2")
    want_z = x.double() @ w.double().T
    assert (z.cpu().double() - want_z).abs().max().item() <= 3e-6 * want_z.abs().max().item()
    r = dict(top=top, scale=1.7)
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    plain.MARGINS = []
    chosen, want = plain.route(x.double(), w[:experts], r)
    sure = plain.MARGINS[0] > 1e-5
    plain.MARGINS = None
    assert sure.float().mean().item() > 0.9
    same = torch.sort(choice.cpu().long(), dim=-1), torch.sort(chosen, dim=-1)
    assert torch.equal(same[0].values[sure], same[1].values[sure])
    got = torch.gather(weight.cpu().double(), 1, same[0].indices)[sure]
    assert (got - torch.gather(want, 1, same[1].indices)[sure]).abs().max().item() <= 2e-6 * want.abs().max().item()
    if groups and 1 < groups[1] < groups[0] and experts // groups[0] > 2:      # the sum of two ranks otherwise than the largest alone
        ops.router(x.to(DEV), w.to(DEV), experts, top, z, other := torch.empty_like(choice), weight, scoring="sigmoid", scale=1.7, groups=groups)
        assert not torch.equal(other, choice)


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
    """``bin/trace_run`` on a Burolorn folder: a prompt in portions beside another request's single tokens."""
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
    """``python -m delta_b200.cli`` on a Burolorn folder: the model class comes from config.json, prompts are scheduled and sampled."""
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

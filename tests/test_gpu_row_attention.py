"""The attention kernels over a cache of rows against the softmax written out in float64: key and value of
different sizes, a value that is the front part of its key (the latent cache), windows, sinks, shuffled pages,
prompt portions beside single tokens.  Queries and keys are made so that one key's score stands out: a key that
a kernel misses (far back, at a page border, at the window's edge) or wrongly sees changes the whole output."""
import math
import random

import pytest
import torch

pytestmark = pytest.mark.gpu

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 2e-5, "bfloat16": 2e-2}


class Ctx:
    """The little of a step's context that the kernel choice reads."""
    def __init__(self, q_lens, dtype, plain):
        self.dtype = DT[dtype]
        self.plain_kernels = {"attention"} if plain else set()
        self.decode_only = all(n == 1 for n in q_lens)
        self.host = dict(q_lens=q_lens)
        self.max_q_len = max(q_lens)
        self.max_seq_len = 0
        self.sm_count = torch.cuda.get_device_properties(0).multi_processor_count
        self._scratch = {}

    def scratch(self, key, shape, dtype, bound=None):
        n = 1
        for s in shape:
            n *= int(s)
        if key not in self._scratch or self._scratch[key].numel() < n:
            self._scratch[key] = torch.empty(max(n, 1), dtype=dtype, device="cuda")
        return self._scratch[key][:n].view(*shape)


def reference(rows, H, KV, dk, dv, scale, window, sink, latent, chunk=None, gates=None):
    out = []
    for (before, n, Q, K, V) in rows:
        Q, K, V = Q.double(), K.double(), V.double()
        o = torch.zeros(n, H, dv, dtype=torch.float64)
        for i in range(n):
            pos = before + i
            lo = max(0, pos - window + 1) if window else 0
            lo = max(lo, pos // chunk * chunk) if chunk else lo
            for h in range(H):
                g = h // (H // KV)
                s = (K[lo:pos + 1, g] @ Q[i, h]) * scale
                m = s.max() if sink is None else torch.maximum(s.max(), sink[h].double())
                e = torch.exp(s - m)
                den = e.sum() + (torch.exp(sink[h].double() - m) if sink is not None else 0.0)
                o[i, h] = (e / den) @ V[lo:pos + 1, g]
        out.append(o)
    o = torch.cat(out)
    return o if gates is None else o * torch.sigmoid(gates.double())[:, :, None]


def run_case(dtype, plain, shape, row_lens, window=None, use_sink=False, latent=False, spikes=(), seed=0, ps=16, chunk=None,
             gated=False):
    """``row_lens``: (tokens cached before the step, new tokens) per batch row.  ``spikes``: (row, query index, key
    position): that query and that key get a large common component."""
    from delta_b200.kernels import ops
    from delta_b200.parts import row_attention
    H, KV, dk, dv = shape
    dt = DT[dtype]
    g = torch.Generator().manual_seed(seed)
    rows = []
    for r, (before, n) in enumerate(row_lens):
        L = before + n
        Q = torch.randn(n, H, dk, generator=g)
        K = torch.randn(L, KV, dk, generator=g)
        V = torch.randn(L, KV, dk if latent else dv, generator=g)
        for (rr, qi, kp) in spikes:
            if rr == r:
                K[kp, :, 0] += 12.0
                Q[qi, :, 0] += 12.0
        Q, K, V = (t.to(dt).float() for t in (Q, K, V))
        if latent:
            V = K[..., :dv].clone()
        rows.append((before, n, Q, K, V))
    scale = 1.0 / math.sqrt(dk)
    sink = (torch.randn(H, generator=g) * 1.5) if use_sink else None
    gates = torch.randn(sum(n for _, n in row_lens), H + 5, generator=g).to(dt) if gated else None      # a head's gate is read in rows with more in them
    want = reference(rows, H, KV, dk, dv, scale, window, sink, latent, chunk, gates[:, :H] if gated else None)
    # the cache, pages handed out in a shuffled order
    row_width = dk if latent else dk + dv
    k_off, v_off = 0, (0 if latent else dk)
    n_pages = sum((b + n + ps - 1) // ps for b, n in row_lens) + 3
    order = list(range(n_pages))
    random.Random(seed).shuffle(order)
    cache = torch.zeros(n_pages, KV, ps, row_width, dtype=dt)
    max_pages = max((b + n + ps - 1) // ps for b, n in row_lens)
    bt = torch.full((len(row_lens), max_pages), -1, dtype=torch.int32)
    nxt = 0
    for r, (before, n, Q, K, V) in enumerate(rows):
        for lp in range((before + n + ps - 1) // ps):
            bt[r, lp] = order[nxt]
            nxt += 1
        for j in range(before + n):
            page, off = int(bt[r, j // ps]), j % ps
            cache[page, :, off, k_off:k_off + dk] = K[j].to(dt)
            if not latent:
                cache[page, :, off, v_off:v_off + dv] = V[j].to(dt)
    for r, (before, _) in enumerate(row_lens):      # pages that no query of the step sees were given back
        lo = max(0, before - window + 1) if window else 0
        lo = max(lo, before // chunk * chunk) if chunk else lo
        bt[r, :lo // ps] = -1
    q = torch.cat([Q.reshape(n, H * dk) for (_, n, Q, _, _) in rows]).to(dt).cuda()
    q_lens = [n for _, n in row_lens]
    starts = [sum(q_lens[:i]) for i in range(len(q_lens))]
    i32 = dict(dtype=torch.int32, device="cuda")
    tok_row = torch.tensor([r for r, n in enumerate(q_lens) for _ in range(n)], **i32)
    tok_pos = torch.tensor([b + i for (b, n) in row_lens for i in range(n)], **i32)
    out = torch.zeros(sum(q_lens), H * dv, dtype=dt, device="cuda")
    err = ops.new_error_record("cuda")
    ctx = Ctx(q_lens, dtype, plain)
    ctx.max_seq_len = max(b + n for b, n in row_lens)
    # (the parameters hold raw addresses: every device tensor stays referenced until the result is read)
    dev = dict(cache=cache.cuda(), block_table=bt.cuda(), row_q_start=torch.tensor(starts, **i32), row_q_len=torch.tensor(q_lens, **i32),
               row_pos_start=torch.tensor([b for b, _ in row_lens], **i32), sink=sink.cuda() if sink is not None else None)
    gates = gates.cuda() if gated else None
    params = ops.row_attn_params(q=q, q_stride=H * dk, q_head_stride=dk, out=out, tok_row=tok_row, tok_pos=tok_pos, H=H, KV=KV, dk=dk,
                                 dv=dv, ps=ps, row_width=row_width, k_off=k_off, v_off=v_off, scale=scale, window=window or 0, chunk=chunk or 0, err=err,
                                 gate_ptr=gates.data_ptr() if gated else None, gate_stride=H + 5,
                                 **dev)
    ctx.err = err
    row_attention.run(ctx, params)
    ops.raise_if_error(err)
    got = out.float().cpu().view(-1, H, dv).double()
    del dev
    worst = (got - want).abs().max().item()
    assert worst <= TOL[dtype] * max(1.0, want.abs().max().item()), f"differs by {worst:.3e}"
    return worst


KERNELS = [("float32", True), ("bfloat16", True), ("bfloat16", False)]     # (precision, the plain kernel)


@pytest.mark.parametrize("dtype,plain", KERNELS)
@pytest.mark.parametrize("shape", [(6, 2, 64, 32), (4, 4, 32, 48), (3, 1, 16, 16), (8, 2, 128, 128)])
def test_prompts_and_single_tokens(dtype, plain, shape):
    run_case(dtype, plain, shape, [(0, 70), (33, 1), (0, 2), (100, 37), (15, 1)], seed=1)
    run_case(dtype, plain, shape, [(130, 1), (0, 1), (17, 1)], use_sink=True, seed=2)
    run_case(dtype, plain, shape, [(0, 150)], use_sink=True, window=40, seed=3, ps=8)


@pytest.mark.parametrize("dtype,plain", KERNELS)
@pytest.mark.parametrize("shape", [(4, 1, 80, 64), (16, 1, 160, 128), (2, 1, 48, 32)])
def test_value_is_the_front_of_the_key(dtype, plain, shape):
    run_case(dtype, plain, shape, [(0, 45), (70, 1), (9, 20)], latent=True, seed=4)
    run_case(dtype, plain, shape, [(200, 1), (31, 1)], latent=True, seed=5)


@pytest.mark.parametrize("dtype,plain", KERNELS)
def test_one_key_that_matters(dtype, plain):
    shape, W, ps = (6, 2, 64, 32), 40, 16
    # in a prompt portion: a far key, keys at both sides of page borders, the first tokens
    for kp in (0, 1, ps - 1, ps, 3 * ps - 1, 3 * ps, 200, 298):
        run_case(dtype, plain, shape, [(150, 150)], spikes=[(0, 149, kp)], seed=kp)
    # decoded alone: the same, among hundreds of keys
    for kp in (0, ps - 1, ps, 255, 256, 400, 519):
        run_case(dtype, plain, shape, [(520, 1), (3, 1)], spikes=[(0, 0, kp)], use_sink=True, seed=kp)
    # the window's edge: the last key inside, the first outside, in a portion and decoded alone
    for inside in (True, False):
        for before, n, qi in ((60, 50, 49), (109, 1, 0), (0, 90, 89), (W - 1, 1, 0), (W, 1, 0)):
            pos = before + qi
            kp = pos - W + 1 if inside else pos - W
            if kp < 0:
                continue
            run_case(dtype, plain, shape, [(before, n), (5, 3)], window=W, use_sink=True, spikes=[(0, qi, kp)], seed=pos)


@pytest.mark.parametrize("dtype,plain", KERNELS)
@pytest.mark.parametrize("shape", [(6, 2, 64, 32), (12, 4, 128, 64), (4, 1, 48, 96), (2, 1, 96, 208), (32, 1, 64, 64)])
def test_chunks_and_gates_of_heads(dtype, plain, shape):
    """Chunks that end inside tiles of queries and of keys, beside a gate per head: portions, single tokens (their keys split over several
    blocks), and both in one step."""
    for chunk in (1, 7, 40, 64, 130):
        run_case(dtype, plain, shape, [(0, 70), (33, 1), (0, 2), (100, 37), (15, 1), (129, 3)], use_sink=True, seed=1, chunk=chunk, gated=True)
        run_case(dtype, plain, shape, [(130, 1), (0, 1), (39, 1), (40, 1)], use_sink=True, seed=2, chunk=chunk, gated=True)
    run_case(dtype, plain, shape, [(0, 150), (500, 1)], seed=3, ps=8, gated=True)
    run_case(dtype, plain, shape, [(700, 1), (640, 1)], seed=3, chunk=600, gated=True)


@pytest.mark.parametrize("dtype,plain", KERNELS)
def test_the_chunks_first_key_and_the_one_before(dtype, plain):
    shape, C = (6, 2, 64, 32), 40
    for before, n, qi in ((60, 50, 19), (79, 1, 0), (0, 130, 79), (0, 130, 80), (40, 1, 0), (41, 5, 3), (599, 1, 0)):
        pos = before + qi
        for kp in (pos // C * C, pos // C * C - 1, pos):
            if kp >= 0:
                run_case(dtype, plain, shape, [(before, n), (5, 3)], chunk=C, use_sink=True, spikes=[(0, qi, kp)], seed=pos)


# ---- the tcgen05 kernel, also for portions shorter than those it is meant for ---------------------------------------------------

TC_SHAPES = [(4, 2, 128, 128), (12, 4, 128, 64), (2, 1, 64, 128), (4, 4, 64, 64), (3, 1, 96, 80), (2, 1, 72, 104), (6, 3, 112, 64)]


@pytest.fixture
def tc_everywhere(monkeypatch):
    from delta_b200.kernels import ops
    from delta_b200.parts import row_attention
    monkeypatch.setattr(row_attention, "TC_MIN_TOKENS", 2)
    calls = []
    real = ops.attention_rows_tc

    def counted(*a):
        calls.append(1)
        return real(*a)
    monkeypatch.setattr(ops, "attention_rows_tc", counted)
    yield calls
    assert calls, "the tcgen05 kernel did not run"


@pytest.mark.parametrize("shape", TC_SHAPES)
def test_tcgen05_portions(tc_everywhere, shape):
    """One tile and many, rows of unequal lengths, contexts before them, windows and chunks that end inside tiles, sinks, gates, pages in runs
    and scattered, pages of several sizes."""
    for ps in ((16, 8, 64) if shape == TC_SHAPES[1] else (16,)):
        run_case("bfloat16", False, shape, [(0, 70), (33, 40), (0, 2), (100, 37), (15, 9)], seed=1, ps=ps)
        run_case("bfloat16", False, shape, [(0, 300), (130, 131)], use_sink=True, gated=True, seed=2, ps=ps)
        run_case("bfloat16", False, shape, [(500, 260), (3, 128)], use_sink=True, window=200, seed=3, ps=ps)
        run_case("bfloat16", False, shape, [(500, 260), (3, 128)], window=33, gated=True, seed=4, ps=ps)
        for chunk in (1, 7, 100, 128, 300):
            run_case("bfloat16", False, shape, [(0, 270), (290, 140), (129, 3)], use_sink=True, gated=True, chunk=chunk, seed=5, ps=ps)


def test_tcgen05_beside_single_tokens(tc_everywhere):
    run_case("bfloat16", False, (12, 4, 128, 64), [(700, 1), (0, 150), (31, 1), (200, 90), (0, 1), (40, 2)], use_sink=True, gated=True, chunk=110, seed=6)
    run_case("bfloat16", False, (8, 2, 128, 128), [(0, 1), (700, 1), (600, 150)], seed=7)


def test_tcgen05_many_pieces(tc_everywhere):
    """More pieces of work than there are multiprocessors: a block takes several, of one tile and of many, one after the other."""
    run_case("bfloat16", False, (16, 4, 128, 64), [(0, 900), (0, 20), (300, 700), (64, 128)], use_sink=True, gated=True, chunk=260, seed=8)
    run_case("bfloat16", False, (16, 4, 64, 128), [(0, 900), (0, 20), (300, 700), (64, 128)], use_sink=True, seed=9)


@pytest.mark.parametrize("kp", [0, 1, 15, 16, 47, 48, 127, 128, 200, 298])
def test_tcgen05_one_key_that_matters(tc_everywhere, kp):
    run_case("bfloat16", False, (4, 2, 128, 64), [(150, 150)], spikes=[(0, 149, kp)], seed=kp)


@pytest.mark.parametrize("before,n,qi", [(60, 50, 19), (0, 130, 79), (0, 130, 80), (41, 5, 3), (119, 128, 0), (120, 128, 127), (0, 128, 40), (0, 128, 39)])
def test_tcgen05_edges_of_chunks_and_windows(tc_everywhere, before, n, qi):
    W, pos = 40, before + qi
    for kp in (pos // W * W, pos // W * W - 1, pos):
        if kp >= 0:
            run_case("bfloat16", False, (4, 2, 128, 64), [(before, n), (5, 3)], chunk=W, use_sink=True, spikes=[(0, qi, kp)], seed=pos)
    for kp in (pos - W + 1, pos - W):
        if kp >= 0:
            run_case("bfloat16", False, (4, 2, 64, 128), [(before, n), (5, 3)], window=W, use_sink=True, spikes=[(0, qi, kp)], seed=pos)

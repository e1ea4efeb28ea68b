"""Burolorn on the CPU: the configuration reader, the specification's tensor list against the names the tests write out on their
own, the states and caches it declares, pages that are given back behind a chunk, and properties of the plain implementation that the
GPU tests lean on."""
import copy
import math

import pytest
import torch

import burolorn_helpers as bh
import plain_burolorn as plain

ALL = ["larger", "wide", "mix", "odd", "one", "sharp", "only_attention", "only_mixing", "only_experts", "only_side"]
F = torch.float64


def build(which):
    import delta_b200.models  # noqa: F401
    from delta_b200.config.registry import architecture_of
    from delta_b200.models import Model
    cfg, W = bh.build(which, 1)
    arch = architecture_of(cfg)
    typed = arch.config_from_dict(cfg)
    return cfg, W, typed, Model(arch.build_spec(typed, None))


@pytest.mark.parametrize("which", ALL)
def test_tensor_list(which):
    _, W, typed, model = build(which)
    first = typed.first_mixing_layer
    unread = set() if first is None else {f"l{first}.mix.vmix"}      # stored, and read by nobody
    names = [s.name for s in model.tensor_specs()]
    assert len(names) == len(set(names))
    assert {s.name: tuple(s.shape) for s in model.tensor_specs()} == {k: tuple(v.shape) for k, v in W.items() if k not in unread}
    assert unread <= set(model.spec.ignorable_tensors)


def test_states_and_caches():
    _, _, _, model = build("mix")
    states = {k: tuple(s.shape) for k, s in model.state_specs().items()}
    assert states == {"run0.conv": (3, 6 * 16 + 3 * 16 + 3 * 24), "run1.conv": (2, 4 * 32 + 2 * 32 + 2 * 16), "run2.conv": (1, 4 * 16 + 4 * 16 + 4 * 8),
                      "run3.conv": (3, 2 * 24 + 24 + 32), "run5.conv": (3, 6 * 16 + 3 * 16 + 3 * 24)}
    assert all(s.dtype == torch.float32 and s.fill == 0.0 for s in model.state_specs().values()) and model.has_run_state()
    caches = model.cache_specs()
    assert {i: (c.page_shape(16), c.chunk, c.window) for i, c in caches.items()} == {
        0: ((3, 16, 40), 24, None), 1: ((2, 16, 48), 50, None), 2: ((4, 16, 24), None, None), 3: ((1, 16, 56), 24, None), 4: ((2, 16, 32), 50, None),
        5: ((3, 16, 40), 24, None)}
    assert caches[0] == caches[5] and caches[0].describe() != caches[2].describe()
    _, _, _, model = build("one")      # one tap carries nothing
    assert list(model.state_specs()) == ["run2.conv"]


def test_constants_reach_the_specification():
    _, _, typed, model = build("mix")
    assert typed.first_mixing_layer == 1 and model.spec.logit_scale == 0.7
    mixers = [b.mixer for b in model.blocks]
    assert [m.value_mix["first"] if m.value_mix else None for m in mixers] == [None, True, False, False, False, None]
    assert [m.taps for m in mixers] == [4, 3, 2, 4, 0, 4] and [m.chunk for m in mixers] == [24, 50, None, 24, 50, 24]
    assert all(m.has_sink and m.head_gate and m.qk_norm_eps == 1e-5 for m in mixers)
    assert [m.position.head_dim if m.position else None for m in mixers] == [8, 32, 6, None, 16, 8] and not mixers[0].position.interleaved
    e = model.blocks[1].feed_forward
    assert (e.experts, e.top, e.groups, e.group_score, e.route_scale, e.scoring, e.normalize, e.shared_gate) == (6, 3, (3, 2), "top2", 1.7, "sigmoid", True, True)
    assert model.blocks[0].feed_forward.is_silu and e.shared.is_silu and model.blocks[2].feed_forward is None
    assert [(b.token_input.index, b.token_input.parts) for b in model.blocks] == [(i, 6) for i in range(6)]
    _, _, typed, model = build("one")
    assert typed.logit_scale == 1.0 and typed.side_dim == 0 and all(b.token_input is None for b in model.blocks)
    assert model.blocks[0].feed_forward.groups is None and model.blocks[0].feed_forward.route_scale == 1.0


def test_config_errors():
    from delta_b200.config.burolorn_config import BurolornConfig
    from delta_b200.config.model_config import ConfigError
    good = bh.config("mix")
    BurolornConfig.from_dict(good)
    for path, value, text in ((("layers", 1, "mixer", "kv_heads"), 3, "multiple"), (("layers", 0, "mixer", "rot", "dims"), 7, "rot.dims"),
                              (("layers", 0, "mixer", "rot", "dims"), 18, "rot.dims"), (("layers", 0, "mixer", "mask", "size"), 0, "chunk"),
                              (("layers", 2, "mixer", "vdim"), 9, "mixed"), (("layers", 1, "mlp", "router", "top"), 7, "top"),
                              (("layers", 1, "mlp", "router", "groups", "count"), 4, "groups"), (("layers", 1, "mlp", "router", "groups", "keep"), 4, "groups"),
                              (("layers", 1, "mlp", "router", "groups", "keep"), 1, "do not hold"), (("layers", 0, "type"), "mamba2", "unknown mixer"),
                              (("layers", 0, "mlp", "kind"), "maxout", "feed-forward kind"), (("layers", 0, "mixer", "dim"), 0, "positive"),
                              (("token_side", "dim"), -3, "token_side")):
        bad = copy.deepcopy(good)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError, match=text):
            BurolornConfig.from_dict(bad)
    for path in (("vocab",), ("norm", "eps"), ("layers", 0, "mixer", "scale"), ("layers", 0, "mixer", "rot", "base"), ("layers", 1, "mlp", "expert", "ff"),
                 ("layers", 0, "mlp", "ff"), ("layers", 0, "mixer", "mask", "size"), ("token_side", "dim")):
        bad = copy.deepcopy(good)
        at = bad
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        if path[-1] in ("size", "dim") and path[0] != "vocab":
            at["other"] = 1
        with pytest.raises(ConfigError, match=path[-1]):
            BurolornConfig.from_dict(bad)


def test_options_that_do_not_go_together():
    from delta_b200.parts.base import PAGE, CacheSpec
    from delta_b200.parts.experts import Experts
    from delta_b200.parts.row_attention import SinkAttention
    base = dict(prefix="x.", width=8, heads=2, kv_heads=1, head_dim=4)
    SinkAttention(**base, conv=3, chunk=5, head_gate=True, qk_norm_eps=1e-5, value_mix=dict(group="v", first=False))
    for bad in (dict(conv=3, bias=True), dict(conv=3, value_from_key=True), dict(value_mix=dict(group="v", first=True), shared_kv=True),
                dict(conv=2, unit_norm_eps=1e-5), dict(conv=2, q_temp=dict(coef=0.1, every=4)), dict(chunk=4, window=4), dict(gate=True, head_gate=True)):
        with pytest.raises(ValueError):
            SinkAttention(**base, **bad)
    with pytest.raises(ValueError):
        CacheSpec((1, PAGE, 8), window=4, chunk=4)
    with pytest.raises(ValueError, match="group"):
        Experts(prefix="x.", width=8, experts=4, top=2, intermediate=4, scoring="sigmoid", groups=(2, 1), group_score="mean")


# ---- pages behind a chunk -----------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("chunk,ps", [(8, 4), (10, 4), (1, 4), (3, 2), (64, 4), (4, 4)])
def test_pages_behind_a_chunk_are_given_back(chunk, ps):
    """After every length the request holds exactly the pages that later queries may read, and the pages fit the next growth."""
    from delta_b200.cache import CacheManager
    from delta_b200.parts.base import PAGE, CacheSpec
    m = CacheManager({0: CacheSpec((1, PAGE, 8), chunk=chunk), 1: CacheSpec((1, PAGE, 8))}, {}, max_slots=2, max_seq_len=64, page_size=ps, num_pages=32,
                     dtype=torch.float32, device="cpu")
    name = CacheSpec((1, PAGE, 8), chunk=chunk).describe()
    for sizes in ([1] * 40, [7, 2, 13, 1, 1, 9, 2], [chunk] * (40 // chunk)):
        slot, n = m.acquire_slot(), 0
        for k in sizes:
            m.grow(slot, n + k)
            n += k
            m.advance(slot, n)
            m.check()
            g = m.groups[name]
            want = list(range((n // chunk * chunk) // ps, -(-n // ps)))
            assert [i for i in range(g.table.shape[1]) if g.table[slot, i] >= 0] == want
        m.release_slot(slot)
        m.check()
        assert all(v == 0 for v in m.pages_in_use().values())


def test_reach_and_first_needed():
    from delta_b200.parts.base import PAGE, CacheSpec
    spec = lambda **k: CacheSpec((1, PAGE, 8), **k)      # noqa: E731
    assert (spec().reach, spec(window=5).reach, spec(chunk=7).reach) == (None, 5, 7)
    assert [spec(window=5).first_needed(n) for n in (0, 4, 5, 9)] == [0, 0, 1, 5]
    assert [spec(chunk=7).first_needed(n) for n in (0, 6, 7, 13, 14)] == [0, 0, 7, 7, 14] and spec().first_needed(99) == 0
    assert len({spec(window=5), spec(chunk=5), spec()}) == 3 and len({s.describe() for s in (spec(window=5), spec(chunk=5), spec())}) == 3


def test_a_pool_that_only_holds_a_few_chunks_takes_a_long_request():
    """Admission counts a chunked group's pages by what it can hold at a time, not by the whole request."""
    from delta_b200.cache import CacheManager
    from delta_b200.engine.scheduler import Scheduler
    from delta_b200.parts.base import PAGE, CacheSpec
    m = CacheManager({0: CacheSpec((1, PAGE, 8), chunk=8)}, {}, max_slots=2, max_seq_len=64, page_size=4, num_pages=6, dtype=torch.float32, device="cpu")
    s = Scheduler(m, max_batch=2, max_tokens_per_step=8)
    assert s._fits_alone(60)
    m2 = CacheManager({0: CacheSpec((1, PAGE, 8))}, {}, max_slots=2, max_seq_len=64, page_size=4, num_pages=6, dtype=torch.float32, device="cpu")
    assert not Scheduler(m2, max_batch=2, max_tokens_per_step=8)._fits_alone(60)


# ---- the plain implementation -------------------------------------------------------------------------------------------------

def test_plain_convolution_and_chunks():
    x = torch.tensor([[1.0, 10.0], [2.0, 20.0], [4.0, 40.0]], dtype=F)
    w = torch.tensor([[0.5, 1.0], [0.0, 2.0]])
    assert torch.equal(plain.causal_conv(x, w), torch.tensor([[1.0, 20.0], [2.5, 40.0], [5.0, 80.0]], dtype=F))
    assert plain.chunk_mask(5, 2).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [0, 0, 1, 0, 0], [0, 0, 1, 1, 0], [0, 0, 0, 0, 1]]
    assert plain.chunk_mask(3, None).int().tolist() == [[1, 0, 0], [1, 1, 0], [1, 1, 1]]
    assert plain.mixed_values(torch.tensor(4.0), torch.tensor(8.0), 0.25).item() == 5.0


def test_plain_sink_rotation_and_gelu():
    w = plain.softmax_with_sink(torch.zeros(1, 2, 2, dtype=F), plain.chunk_mask(2, None)[None], torch.tensor([math.log(3.0)]))
    assert torch.allclose(w[0], torch.tensor([[0.25, 0.0], [0.2, 0.2]], dtype=F), atol=1e-6)
    x = torch.randn(5, 2, 6, dtype=F)
    y = plain.rotate_halves(x, torch.arange(5), dict(base=100.0, dims=4))
    assert torch.equal(y[..., 4:], x[..., 4:]) and torch.equal(y[0], x[0])
    assert torch.allclose(y[3, :, 0], x[3, :, 0] * math.cos(3.0) - x[3, :, 2] * math.sin(3.0))
    assert torch.allclose(y[3, :, 3], x[3, :, 3] * math.cos(0.3) + x[3, :, 1] * math.sin(0.3))
    z = torch.tensor([-2.0, 0.0, 1.5], dtype=F)
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))


def test_plain_router_by_hand():
    """Six experts in three groups of two, two kept: the group with the largest single score is left out, because the sum of its two is the
    smallest; the weights are the chosen scores over their sum, times the scale."""
    z = torch.tensor([2.0, -9.0, 1.0, 0.5, 1.2, 0.1], dtype=F)
    h, W = torch.eye(6, dtype=F)[:1], torch.zeros(6, 6, dtype=F)
    W[:, 0] = z
    s = torch.sigmoid(z)
    chosen, weight = plain.route(h, W, dict(top=3, groups=dict(count=3, keep=2), scale=2.0))
    assert chosen.tolist() == [[4, 2, 3]] and torch.allclose(weight[0], 2.0 * s[[4, 2, 3]] / s[[4, 2, 3]].sum())
    chosen, weight = plain.route(h, W, dict(top=2))
    assert chosen.tolist() == [[0, 4]] and torch.allclose(weight[0], s[[0, 4]] / s[[0, 4]].sum())
    chosen, _ = plain.route(h, W, dict(top=2, groups=dict(count=6, keep=2)))      # groups of one: their only score
    assert chosen.tolist() == [[0, 4]]


@pytest.mark.parametrize("which", ["mix", "odd", "only_attention", "only_mixing", "only_side"])
def test_plain_model_is_causal(which):
    """A changed token changes nothing before it, and the token behind it."""
    cfg, W = bh.build(which, 3)
    toks = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(1)).tolist()
    other = list(toks)
    other[20] = (other[20] + 1) % cfg["vocab"]
    a, b = plain.forward(cfg, W, toks)[0], plain.forward(cfg, W, other)[0]
    assert torch.allclose(a[:20], b[:20], atol=1e-12)
    assert (a[21] - b[21]).abs().max().item() > 1e-4 * a.abs().max().item()


@pytest.mark.parametrize("what", ["sink", "chunk", "rot", "vmix", "conv", "gate", "side", "groups", "scale", "sg", "k.norm"])
def test_every_mechanism_shows_in_the_plain_logits(what):
    """Leaving one mechanism out (in the plain implementation's inputs) moves the logits of the mixed test model by far more than the bound the
    engine is held to."""
    cfg, W = bh.build("mix", 3)
    toks = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(2)).tolist()
    ref = plain.forward(cfg, W, toks)[0]
    c2, W2 = copy.deepcopy(cfg), dict(W)
    for i, L in enumerate(c2["layers"]):
        m = L["mixer"]
        if what == "sink":
            W2[f"l{i}.mix.sink"] = torch.full_like(W2[f"l{i}.mix.sink"], -99.0)
        elif what == "chunk" and m.get("mask"):
            m["mask"]["size"] += 1
        elif what == "rot" and m.get("rot"):
            m["rot"]["base"] *= 2
        elif what == "vmix" and m.get("v_mix"):
            W2[f"l{i}.mix.vmix"] = torch.zeros(())
        elif what == "conv" and m.get("conv"):
            W2[f"l{i}.mix.v.conv"] = W2[f"l{i}.mix.v.conv"].roll(1, dims=1)
        elif what == "gate":
            W2[f"l{i}.mix.g"] = torch.zeros_like(W2[f"l{i}.mix.g"])
        elif what == "side":
            W2[f"l{i}.side.proj"] = torch.zeros_like(W2[f"l{i}.side.proj"])
        elif what == "k.norm":
            W2[f"l{i}.mix.k.norm"] = torch.ones_like(W2[f"l{i}.mix.k.norm"])
        elif L.get("mlp") and L["mlp"]["kind"] == "moe":
            if what == "groups":
                L["mlp"]["router"].pop("groups", None)
            elif what == "scale":
                L["mlp"]["router"].pop("scale", None)
            elif what == "sg" and L["mlp"].get("shared"):
                W2[f"l{i}.mlp.shared.sg"] = torch.zeros_like(W2[f"l{i}.mlp.shared.sg"])
    moved = (plain.forward(c2, W2, toks)[0] - ref).abs().max().item() / ref.abs().max().item()
    assert moved > 0.02, moved

"""Vazunex on the CPU: the configuration reader (with sizes that only the tensors' shapes give), the specification's tensor list
against the names the tests write out on their own, the states and caches it declares, and properties of the plain implementation
that the GPU tests lean on."""
import copy
import math

import pytest
import torch

import plain_vazunex as plain
import vazunex_helpers as vh

ALL = ["larger", "wide", "mix", "odd", "one", "sharp", "only_delta", "only_ssd", "only_latent", "only_experts"]
F = torch.float64


def build(which):
    import delta_b200.models  # noqa: F401
    from delta_b200.config.registry import architecture_of
    from delta_b200.models import Model
    cfg, W = vh.build(which, 1)
    arch = architecture_of(cfg)
    typed = arch.config_from_dict(arch.sizes_from_shapes(cfg, {k: tuple(v.shape) for k, v in W.items()}))
    return cfg, W, typed, Model(arch.build_spec(typed, None))


@pytest.mark.parametrize("which", ALL)
def test_tensor_list(which):
    _, W, _, model = build(which)
    assert {s.name: tuple(s.shape) for s in model.tensor_specs()} == {k: tuple(v.shape) for k, v in W.items()}


def test_ranks_come_from_the_shapes_or_from_the_file():
    from delta_b200.config.model_config import ConfigError
    from delta_b200.config.vazunex_config import VazunexConfig, sizes_from_shapes
    cfg, W, typed, _ = build("mix")
    assert [(L.mixer["decay_rank"], L.mixer["gate_rank"]) for L in typed.layers if L.type == "channel_delta"] == [(12, 20), (8, 8)]
    with pytest.raises(ConfigError, match="decay_rank"):
        VazunexConfig.from_dict(cfg)
    given = copy.deepcopy(cfg)
    for L in given["layers"]:
        if L["type"] == "channel_delta":
            L["mixer"].update(decay_rank=3, gate_rank=5)
    assert VazunexConfig.from_dict(given).layers[2].mixer["gate_rank"] == 5
    assert sizes_from_shapes(given, {k: tuple(v.shape) for k, v in W.items()})["layers"][2]["mixer"]["gate_rank"] == 5      # config.json wins


def test_states_and_caches():
    _, _, _, model = build("mix")
    by_run = {}
    for k, s in model.state_specs().items():
        by_run.setdefault(k.split(".")[0], {})[k.split(".", 1)[1]] = tuple(s.shape)
        assert s.dtype == torch.float32 and s.fill == 0.0
    assert by_run == {"run0": {"conv": (3, 6 * 16 + 2 * 2 * 24), "ssd": (6, 16, 24)}, "run2": {"conv": (3, 2 * 3 * 16 + 6 * 24), "delta": (6, 24, 16)},
                      "run4": {"conv": (1, 4 * 40 + 2 * 4 * 12), "ssd": (4, 40, 12)}, "run5": {"conv": (2, 2 * 24 + 4 * 16), "delta": (4, 16, 24)}}
    caches = model.cache_specs()
    assert {i: (c.page_shape(16), c.window) for i, c in caches.items()} == {1: ((1, 16, 48), 21), 3: ((1, 16, 40), 50)}
    assert model.has_run_state()
    _, _, _, model = build("one")      # no window: every token is kept; one tap: no inputs are carried, the state has a row nobody reads
    assert {i: c.window for i, c in model.cache_specs().items()} == {2: 1, 3: None}
    assert tuple(model.state_specs()["run0.conv"].shape) == (1, 10)


def test_constants_reach_the_specification():
    _, _, typed, model = build("mix")
    assert [b.update_scale for b in model.blocks] == [0.4] * 6 and model.spec.logit_scale == 0.7
    assert all(n.weight_offset == 1.0 for n in (model.final_norm, model.stream.start_norm, model.blocks[0].norm1, model.blocks[0].norm2))
    e = model.blocks[0].feed_forward
    assert (e.experts, e.identity, e.outputs, e.groups, e.top, e.route_scale, e.normalize, e.scoring) == (7, 2, 9, (3, 2), 3, 1.7, False, "softmax_all")
    _, _, typed, model = build("one")
    assert (typed.residual_mult, typed.logit_scale) == (1.0, 1.0) and model.blocks[0].feed_forward.groups is None
    a = model.blocks[2].mixer
    assert a.window == 1 and a.has_sink and a.has_gate and not a.position.interleaved


def test_config_errors():
    from delta_b200.config.model_config import ConfigError
    from delta_b200.config.vazunex_config import VazunexConfig, sizes_from_shapes
    cfg, W = vh.build("mix", 1)
    good = sizes_from_shapes(cfg, {k: tuple(v.shape) for k, v in W.items()})
    VazunexConfig.from_dict(good)
    for path, value, text in ((("layers", 2, "mixer", "kv_heads"), 4, "multiple"), (("layers", 0, "mixer", "groups"), 4, "groups"),
                              (("layers", 0, "mixer", "norm_groups"), 7, "equal parts"), (("layers", 0, "mixer", "conv"), 0, "positive"),
                              (("layers", 1, "mixer", "rot", "dims"), 7, "rot.dims"), (("layers", 1, "mixer", "rot", "dims"), 10, "rot.dims"),
                              (("layers", 1, "mixer", "mask", "size"), 0, "window"), (("layers", 0, "mlp", "router", "top"), 10, "top"),
                              (("layers", 0, "mlp", "router", "groups", "count"), 2, "groups"), (("layers", 0, "mlp", "router", "groups", "keep"), 4, "groups"),
                              (("layers", 2, "mlp", "router", "top"), 4, "do not hold"), (("layers", 0, "type"), "mamba1", "unknown mixer"),
                              (("layers", 0, "mlp", "kind"), "dense", "feed-forward kind")):
        bad = copy.deepcopy(good)
        at = bad
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(ConfigError, match=text):
            VazunexConfig.from_dict(bad)
    for path in (("vocab",), ("norm", "eps"), ("layers", 0, "mixer", "state"), ("layers", 1, "mixer", "rot"), ("layers", 0, "mlp", "expert", "ff")):
        bad = copy.deepcopy(good)
        at = bad
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        with pytest.raises(ConfigError, match=path[-1]):
            VazunexConfig.from_dict(bad)


def test_expert_options_that_do_not_go_together():
    from delta_b200.parts.experts import Experts
    base = dict(prefix="x.", width=8, experts=4, top=2, intermediate=4)
    Experts(**base, scoring="softmax_all", normalize=False, correction=True, identity=2, groups=(3, 2))
    for bad in (dict(scoring="softmax", groups=(2, 1)), dict(scoring="softmax_all", groups=(3, 1)), dict(scoring="softmax_all", groups=(4, 1)),
                dict(scoring="softmax", normalize=False), dict(scoring="none"), dict(scoring="softmax_all", identity=1, weight_input=True)):
        with pytest.raises(ValueError):
            Experts(**base, **bad)


# ---- the plain implementation -------------------------------------------------------------------------------------------------

def test_plain_convolution_and_norms():
    x = torch.tensor([[1.0, 10.0], [2.0, 20.0], [4.0, 40.0]], dtype=F)
    w = torch.tensor([[0.5, 1.0], [0.0, 2.0]])
    assert torch.equal(plain.causal_conv(x, w, torch.tensor([0.25, 0.0])), torch.tensor([[1.25, 20.0], [2.75, 40.0], [5.25, 80.0]], dtype=F))
    assert torch.allclose(plain.offset_norm(x, torch.zeros(2), 0.0).pow(2).mean(-1), torch.ones(3, dtype=F))
    assert torch.allclose(plain.unit_vector(x).pow(2).sum(-1), torch.ones(3, dtype=F), atol=1e-6)


def test_plain_recurrences_by_hand():
    """One head, one key channel, one value: the delta rule reads what it wrote, and a second write of the same key replaces it; the
    state-space recurrence decays and adds."""
    one = lambda *v: torch.tensor(v, dtype=F).view(-1, 1, 1)      # noqa: E731
    o = plain.delta_recurrence(one(1, 1, 1), one(1, 1, 1), one(3, 5, 0), torch.tensor([[1.0], [1.0], [0.0]], dtype=F), one(1, 1, 0.5))
    assert o.flatten().tolist() == [3.0, 5.0, 2.5]
    y = plain.ssd_recurrence(one(2, 0), one(1, 1), one(1, 3), torch.tensor([[0.5], [1.0]], dtype=F), torch.tensor([math.log(2.0)], dtype=F), torch.tensor([10.0], dtype=F))
    assert y.flatten().tolist() == pytest.approx([0.5 * 2 + 20, 3 * 0.5 * 1.0], abs=1e-12)


def test_plain_router_by_hand():
    """Six outputs in three groups of two, two groups kept: an output of a dropped group is not chosen although its choice score is larger
    than a chosen one's; negative choice scores are no reason to leave a group out; the weights are the scores without the correction."""
    h = torch.eye(6, dtype=F)[:1]
    want_s = torch.softmax(torch.tensor([3.0, 0.0, 2.0, 1.9, 2.5, -1.0], dtype=F), 0)
    W = torch.zeros(6, 6, dtype=F)
    W[:, 0] = torch.tensor([3.0, 0.0, 2.0, 1.9, 2.5, -1.0], dtype=F)
    corr = torch.full((6,), -0.9, dtype=F)
    chosen, weight = plain.route(h, W, corr, dict(top=3, groups=dict(count=3, keep=2), scale=2.0))
    assert chosen.tolist() == [[0, 4, 1]] and torch.allclose(weight[0], 2.0 * want_s[[0, 4, 1]])
    chosen, _ = plain.route(h, W, corr, dict(top=3))
    assert chosen.tolist() == [[0, 4, 2]]
    corr[3] += 0.5                                                  # the correction alone lifts the middle group to the top
    chosen, weight = plain.route(h, W, corr, dict(top=2, groups=dict(count=3, keep=1)))
    assert chosen.tolist() == [[3, 2]] and torch.allclose(weight[0], want_s[[3, 2]])


def test_plain_window_sink_and_rotation():
    assert plain.window_mask(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    assert plain.window_mask(3, None).int().tolist() == [[1, 0, 0], [1, 1, 0], [1, 1, 1]]
    w = plain.softmax_with_sink(torch.zeros(1, 2, 2, dtype=F), plain.window_mask(2, None)[None], torch.tensor([math.log(3.0)]))
    assert torch.allclose(w[0], torch.tensor([[0.25, 0.0], [0.2, 0.2]], dtype=F), atol=1e-6)
    x = torch.randn(5, 6, dtype=F)
    y = plain.rotate_halves(x, torch.arange(5), dict(base=100.0, dims=4))
    assert torch.equal(y[:, 4:], x[:, 4:]) and torch.equal(y[0], x[0])
    assert torch.allclose(y[3, 0], x[3, 0] * math.cos(3.0) - x[3, 2] * math.sin(3.0)) and torch.allclose(y[3, 3], x[3, 3] * math.cos(0.3) + x[3, 1] * math.sin(0.3))


@pytest.mark.parametrize("which", ["mix", "odd", "only_delta", "only_ssd"])
def test_plain_model_is_causal_and_remembers(which):
    """A changed token changes nothing before it, and something far behind it (the recurrences carry it)."""
    cfg, W = vh.build(which, 3)
    toks = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(1)).tolist()
    other = list(toks)
    other[20] = (other[20] + 1) % cfg["vocab"]
    a, b = plain.forward(cfg, W, toks)[0], plain.forward(cfg, W, other)[0]
    assert torch.allclose(a[:20], b[:20], atol=1e-12)
    assert (a[-1] - b[-1]).abs().max().item() > 1e-4 * a.abs().max().item()

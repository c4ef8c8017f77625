"""Lasupel without a GPU: configuration, spec, tensor names, cache and state bookkeeping, the oracle's own parts."""

import json
from dataclasses import replace

import pytest
import torch

import plain_lasupel as plain
from lasupel_configs import LASUPEL_CONFIGS, LASUPEL_SEEDS, tensors_of
from tinyvllm_b200.cache.manager import CacheManager
from tinyvllm_b200.cache.storage import CacheStorage, group_runs
from tinyvllm_b200.config.registry import ConfigError, parse_model_config
from tinyvllm_b200.engine.model import Model
from tinyvllm_b200.models import LasupelConfig
from tinyvllm_b200.parts.base import KVNeed, kv_need, state_needs
from tinyvllm_b200.weights.loader import WeightsError, bind_tensors
from tinyvllm_b200.weights.random_init import random_tensors

F64 = torch.float64


@pytest.mark.parametrize("name", sorted(LASUPEL_CONFIGS))
def test_config_round_trip_and_registry(name):
    config = LASUPEL_CONFIGS[name]
    data = json.loads(json.dumps(config.to_json()))
    assert data["architecture"] == "Lasupel"
    again = parse_model_config(data)
    assert isinstance(again, LasupelConfig) and again == config and again.to_json() == data


def test_what_may_be_left_out():
    data = LASUPEL_CONFIGS["a"].to_json()
    data["layers"][1]["mlp"]["router"].pop("groups")
    data["layers"][1]["mixer"].pop("rot"), data["layers"][3]["mixer"].pop("rot")
    data["layers"][1]["mixer"].pop("mask")
    data["layers"][2]["mlp"] = None
    data.pop("embedding")
    config = parse_model_config(data)
    assert config.embedding_scale == 1.0 and config.layers[2].mlp is None
    assert (config.layers[1].mlp.groups, config.layers[1].mlp.keep) == (1, 1)
    assert config.layers[1].mixer.window is None and config.layers[1].mixer.rot_dims == 0


def test_config_refusals():
    good = LASUPEL_CONFIGS["a"].to_json()
    for change in (lambda d: d.pop("norm"), lambda d: d.pop("width"), lambda d: d["norm"].update(eps=0.0),
                   lambda d: d.update(vocab=0), lambda d: d["embedding"].update(scale="2"),
                   lambda d: d["layers"][0].update(type="scan"),
                   lambda d: d["layers"][0]["mixer"].pop("blocks"),
                   lambda d: d["layers"][0]["mixer"].update(blocks=5),
                   lambda d: d["layers"][0]["mixer"].update(conv=0),
                   lambda d: d["layers"][1]["mixer"].pop("scale"),
                   lambda d: d["layers"][1]["mixer"].update(heads=3),
                   lambda d: d["layers"][1]["mixer"]["mask"].update(size=0),
                   lambda d: d["layers"][1]["mixer"]["rot"].update(dims=18),
                   lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7),
                   lambda d: d["layers"][1]["mlp"].update(kind="sparse"),
                   lambda d: d["layers"][1]["mlp"]["expert"].pop("limit"),
                   lambda d: d["layers"][1]["mlp"]["router"].update(top=5),         # more than the kept groups hold
                   lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(count=4),
                   lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(keep=4),
                   lambda d: d["layers"][2]["mixer"].update(kv_heads=3),
                   lambda d: d["layers"][2]["mixer"].pop("vdim"),
                   lambda d: d["layers"][3]["mixer"].update(kv_from=3),
                   lambda d: d["layers"][3]["mixer"].update(kv_from=0),             # not attention
                   lambda d: d["layers"][3]["mixer"].update(kv_from=-1),
                   lambda d: d["layers"][3]["mixer"].update(dim=32),
                   lambda d: d["layers"][3]["mixer"].update(kv_heads=4)):
        data = json.loads(json.dumps(good))
        change(data)
        with pytest.raises(ConfigError):
            parse_model_config(data)
    chained = LASUPEL_CONFIGS["c"].to_json()
    chained["layers"][4]["mixer"]["kv_from"] = 3                                    # has no keys of its own
    with pytest.raises(ConfigError):
        parse_model_config(chained)


@pytest.mark.parametrize("name", sorted(LASUPEL_CONFIGS))
def test_the_model_declares_exactly_the_checkpoint_tensors(name):
    config = LASUPEL_CONFIGS[name]
    model = Model(config.to_spec(), device="cpu", dtype=torch.float32)
    declared, shapes, optional = {}, {}, set()
    for _, spec in model.param_targets():
        for source in spec.sources:
            declared[source.name] = declared.get(source.name, 0) + 1
            shapes[source.name] = (source.rows,) + (tuple(spec.shape[1:]) if source.cols is None else (source.cols,))
            if spec.optional:
                optional.add(source.name)
    tensors = tensors_of(config, LASUPEL_SEEDS[name])
    assert all(count == 1 for count in declared.values())
    # a layer without a feed-forward may come with its second norm or without
    assert optional == {f"l{i}.norm2" for i, layer in enumerate(config.layers) if layer.mlp is None}
    assert set(declared) - optional == set(tensors)
    assert all(tuple(tensors[n].shape) == shapes[n] for n in tensors)


@pytest.mark.parametrize("name", sorted(LASUPEL_CONFIGS))
def test_weights_are_bound_and_packed(name):
    """Every tensor finds its place: packed input projections hold the mixer's rows in order (zeros up to a multiple of
    8), both gates of a block stand in one matrix, taps by age with zeros in front, decays and rates as the kernels
    read them."""
    config = LASUPEL_CONFIGS[name]
    tensors = tensors_of(config, LASUPEL_SEEDS[name])
    model = Model(config.to_spec(), device="cpu", dtype=torch.float32)
    bind_tensors(model.param_targets(), tensors, dtype=torch.float32, device="cpu")
    model._after_binding()
    for index, (layer, block) in enumerate(zip(config.layers, model.blocks)):
        at, mixer, m = f"l{index}.mix.", block.mixer, layer.mixer
        if layer.type == "attention":
            names = ("q",) if m.kv_from is not None else ("q", "k", "v")
            assert torch.equal(mixer.in_weight, torch.cat([tensors[at + n] for n in names]))
            continue
        taps = m.conv
        if layer.type == "rglru":
            assert torch.equal(mixer.in_weight, torch.cat([tensors[at + "x"], tensors[at + "y"]]))
            size = m.width // m.blocks
            assert torch.equal(mixer.gate_weight[:, :size], tensors[at + "ra"])
            assert torch.equal(mixer.gate_weight[:, size:], tensors[at + "ri"])
            assert torch.equal(mixer.r_bias, tensors[at + "ra.b"].flatten())
            assert torch.allclose(mixer.decay, -8.0 * torch.nn.functional.softplus(tensors[at + "lam"]))
            want = tensors[at + "conv"]
        else:
            want = torch.cat([tensors[at + n] for n in ("q", "k", "v", "g", "b", "a")])
            assert torch.equal(mixer.in_weight[:want.shape[0]], want) and not mixer.in_weight[want.shape[0]:].any()
            assert mixer.in_weight.shape[0] % 8 == 0
            assert torch.allclose(mixer.rate, -torch.exp(tensors[at + "A_log"]))
            want = torch.cat([tensors[at + n + ".conv"] for n in ("q", "k", "v")])
        assert torch.equal(mixer.conv_by_tap[-taps:], want.t())
        assert not mixer.conv_by_tap[:-taps].any() and mixer.conv_by_tap.shape[0] >= 2
    model._after_binding()                                   # a second time changes nothing


def test_a_second_norm_that_nothing_reads_may_be_there():
    config = LASUPEL_CONFIGS["d"]
    tensors = tensors_of(config, 1)
    tensors["l0.norm2"] = torch.ones(config.width)
    model = Model(config.to_spec(), device="cpu", dtype=torch.float32)
    bind_tensors(model.param_targets(), tensors, dtype=torch.float32, device="cpu")
    tensors["l0.norm3"] = torch.ones(config.width)
    with pytest.raises(WeightsError, match="l0.norm3"):
        bind_tensors(Model(config.to_spec(), device="cpu", dtype=torch.float32).param_targets(), tensors,
                     dtype=torch.float32, device="cpu")


def test_random_weights_cover_every_tensor():
    for name in ("a", "b"):
        model = Model(LASUPEL_CONFIGS[name].to_spec(), device="cpu", dtype=torch.float32)
        targets = model.param_targets()
        bind_tensors(targets, random_tensors(targets, 3), dtype=torch.float32, device="cpu")
        model._after_binding()


# ------------------------------------------------------------------- caches
@pytest.mark.parametrize("name", sorted(LASUPEL_CONFIGS))
def test_every_layer_has_the_pages_and_states_it_needs(name):
    config = LASUPEL_CONFIGS[name]
    model = Model(config.to_spec(), device="cpu", dtype=torch.bfloat16)
    needs, sources = model.cache_needs(), model.cache_sources()
    groups, where = group_runs(needs, sources)
    for index, (layer, need) in enumerate(zip(config.layers, needs)):
        m = layer.mixer
        if layer.type == "attention":
            assert kv_need(need) == KVNeed(m.kv_heads, m.dim, m.window, m.vdim, 0) and not state_needs(need)
            assert where[index] == where[m.kv_from if m.kv_from is not None else index]
            continue
        state, conv = state_needs(need)
        assert kv_need(need) is None and state.dtype == conv.dtype == torch.float32
        assert state.shape == ((m.width,) if layer.type == "rglru" else (m.heads, m.dim, m.vdim))
        assert conv.shape[0] >= max(1, m.conv - 1)
    storage = CacheStorage(groups, where, needs, page_size=4, pages_per_group=3, num_state_slots=2, dtype=torch.float32,
                           device="cpu", other_states=model.other_states())
    assert len(storage.state) == 2 * sum(layer.type != "attention" for layer in config.layers)
    owners = [i for i, layer in enumerate(config.layers) if layer.type == "attention" and layer.mixer.kv_from is None]
    assert sorted(run for group in groups for run in group.runs) == owners


def test_a_shared_cache_is_kept_for_the_widest_window():
    own = KVNeed(2, 16, 24)
    cases = ((8, 24), (24, 24), (75, 75), (None, None))
    for window, kept in cases:
        groups, where = group_runs([own, KVNeed(2, 16, window)], [None, 0])
        assert groups[0].window == kept and where == {0: (0, 0), 1: (0, 0)}
    groups, where = group_runs([own, KVNeed(2, 16, 24), KVNeed(2, 16, 30), KVNeed(2, 16, 90)], [None, None, 1, 1])
    # the layer whose cache is kept longer has a group of its own
    assert [g.window for g in groups] == [24, 90] and where[3] == where[1] == (1, 0)
    assert group_runs([KVNeed(2, 16, None), KVNeed(2, 16, 5)], [None, 0])[0][0].window is None
    for other in (KVNeed(1, 16, 24), KVNeed(2, 32, 24), KVNeed(2, 16, 24, 8), KVNeed(2, 16, 24, 16, 0, 0)):
        with pytest.raises(ValueError):
            group_runs([own, other], [None, 0])


def test_pages_outlive_the_narrower_window():
    """A request of 40 tokens over pages of 4: with a reader that sees 17 tokens behind a layer that sees 6, pages go
    back only behind the wider window."""
    for windows, first in (((6, 17), 24), ((6, 3), 35), ((6, None), 0)):
        groups, _ = group_runs([KVNeed(1, 8, windows[0]), KVNeed(1, 8, windows[1])], [None, 0])
        manager = CacheManager(groups, 4, 12, 1)
        manager.open("r")
        for count in (30, 1, 1, 8):
            plan = manager.plan([("r", count)])
            assert plan is not None
            manager.commit(plan)
        table = manager.block_table("r", 0)
        assert [page >= 0 for page in table] == [4 * i + 3 >= first for i in range(10)]
        manager.close("r")
        manager.check()
        assert manager.free_pages(0) == 12


# -------------------------------------------------------------- the oracle's own parts
def test_the_oracles_softmax_has_one_more_term():
    s = torch.tensor([[0.0, 1.0, -torch.inf], [-40.0, -41.0, -39.0]], dtype=F64)
    e = torch.exp(s)
    assert torch.allclose(plain.softmax_with_sink(s), e / (1.0 + e.sum(-1, keepdim=True)))
    assert plain.softmax_with_sink(s)[1].sum() < 1e-15
    big = plain.softmax_with_sink(torch.tensor([[900.0, 899.0]], dtype=F64))
    assert torch.allclose(big, torch.softmax(torch.tensor([[1.0, 0.0]], dtype=F64), -1))


def test_the_oracles_windows_and_rotation():
    at = torch.arange(9)
    seen = plain.visible(at, at, 3)
    assert [seen[6, j].item() for j in range(9)] == [False] * 4 + [True] * 3 + [False] * 2
    assert plain.visible(at, at, None)[8].all() and plain.visible(at, at, 1).equal(torch.eye(9, dtype=torch.bool))
    g = torch.Generator().manual_seed(1)
    x = torch.randn(9, 2, 10, generator=g, dtype=F64)
    turned = plain.rotate_halves(x, at, {"dims": 6, "base": 50.0})
    assert torch.equal(turned[..., 6:], x[..., 6:]) and torch.allclose(turned[0], x[0])
    angle = 4 * 50.0 ** (-2.0 / 6)
    want = torch.cos(torch.tensor(angle, dtype=F64)) * x[4, 1, 1] - torch.sin(torch.tensor(angle, dtype=F64)) * x[4, 1, 4]
    assert torch.allclose(turned[4, 1, 1], want)
    # a rotation moves no length: normed before or behind it, the heads are the same
    assert torch.allclose(plain.over_rms(turned, 1e-5),
                          plain.rotate_halves(plain.over_rms(x, 1e-5), at, {"dims": 6, "base": 50.0}))


def test_the_oracles_router():
    """The best groups are those with the largest single score: a group of two good experts loses to one with the best."""
    z = torch.log(torch.tensor([[0.22, 0.23, 0.01, 0.30, 0.14, 0.10]], dtype=F64))
    w = plain.chosen_weights(z, 1, {"count": 3, "keep": 1})
    assert torch.allclose(w, torch.tensor([[0, 0, 0, 0.30, 0, 0]], dtype=F64))
    w = plain.chosen_weights(z, 3, {"count": 3, "keep": 2})
    assert torch.allclose(w, torch.tensor([[0.22, 0.23, 0, 0.30, 0, 0]], dtype=F64))
    w = plain.chosen_weights(z, 4, None)
    assert torch.allclose(w, torch.tensor([[0.22, 0.23, 0, 0.30, 0.14, 0]], dtype=F64))


def test_the_oracles_delta_rule_replaces_what_a_key_holds():
    g = torch.Generator().manual_seed(2)
    k = plain.unit(torch.randn(1, 1, 6, generator=g, dtype=F64)).repeat(3, 1, 1)
    v = torch.randn(3, 1, 4, generator=g, dtype=F64)
    one = torch.ones(3, 1, dtype=F64)
    o, state = plain.delta_rule(k, k, v, one, one)
    assert torch.allclose(o, v, atol=1e-5)                       # a full step leaves the newest value alone
    _, kept = plain.delta_rule(k[:1], k[:1], v[:1], 0.5 * one[:1], 0.0 * one[:1], state)
    assert torch.allclose(kept, 0.5 * state)
    half, _ = plain.delta_rule(k[:2], k[:2], v[:2], one[:2], 0.5 * one[:2])
    assert torch.allclose(half[1], 0.25 * v[0] + 0.5 * v[1], atol=1e-5)


def test_the_oracles_recurrences_carry_their_states():
    """Cut in two, the recurrent unit and the delta rule give what they give whole; the inputs before a start are zeros,
    not biases."""
    g = torch.Generator().manual_seed(3)
    shapes = {"m.y": (6, 5), "m.y.b": (6,), "m.x": (6, 5), "m.x.b": (6,), "m.conv": (6, 3), "m.conv.b": (6,),
              "m.ra": (2, 3, 3), "m.ra.b": (2, 3), "m.ri": (2, 3, 3), "m.ri.b": (2, 3), "m.lam": (6,), "m.o": (5, 6),
              "n.q": (3, 5), "n.q.conv": (3, 3), "n.k": (3, 5), "n.k.conv": (3, 3), "n.v": (8, 5), "n.v.conv": (8, 3),
              "n.b": (2, 5), "n.a": (2, 5), "n.A_log": (2,), "n.dt_bias": (2,), "n.g": (8, 5), "n.norm": (4,), "n.o": (5, 8)}
    w = {name: torch.randn(shape, generator=g, dtype=F64) for name, shape in shapes.items()}
    h = torch.randn(9, 5, generator=g, dtype=F64)
    whole, state, tail = plain.rglru(h, w, "m", None)
    first, s1, t1 = plain.rglru(h[:4], w, "m", None)
    second, s2, t2 = plain.rglru(h[4:], w, "m", None, state=s1, before=t1)
    assert torch.allclose(torch.cat([first, second]), whole) and torch.allclose(s2, state) and torch.allclose(t2, tail)
    x = h @ w["m.x"].T + w["m.x.b"]
    u, _ = plain.causal_convolution(x, w["m.conv"])
    assert torch.allclose(u[0], w["m.conv"][:, 2] * x[0])
    assert torch.allclose(u[1], w["m.conv"][:, 2] * x[1] + w["m.conv"][:, 1] * x[0])
    gate = plain.block_gate(u, w["m.ra"], w["m.ra.b"])
    assert torch.allclose(gate[4, 3:], torch.sigmoid(w["m.ra"][1] @ u[4, 3:] + w["m.ra.b"][1]))
    mixer = {"heads": 2, "kv_heads": 1, "dim": 3, "vdim": 4}
    whole, state, _ = plain.delta(h, w, "n", mixer, 1e-6)
    first, s1, t1 = plain.delta(h[:4], w, "n", mixer, 1e-6)
    second, s2, _ = plain.delta(h[4:], w, "n", mixer, 1e-6, state=s1, before=t1)
    assert torch.allclose(torch.cat([first, second]), whole) and torch.allclose(s2, state)


def test_the_oracles_experts_are_clipped():
    w = {"e.gate": torch.tensor([[1.0]], dtype=F64), "e.up": torch.tensor([[1.0]], dtype=F64),
         "e.down": torch.tensor([[1.0]], dtype=F64)}
    for h, g, u in ((5.0, 2.0, 2.0), (-5.0, -5.0, -2.0), (0.5, 0.5, 0.5)):
        want = g / (1.0 + torch.exp(torch.tensor(-1.702 * g, dtype=F64))) * (u + 1.0)
        assert torch.allclose(plain.expert(torch.tensor([[h]], dtype=F64), w, "e", 2.0), want)


def test_the_spec_names_the_run_whose_cache_is_read():
    config = LASUPEL_CONFIGS["c"]
    assert [step.cache_from for step in config.to_spec().order] == [None, None, None, 1, 1]
    alone = replace(config, layers=config.layers[:3])
    assert all(step.cache_from is None for step in alone.to_spec().order)

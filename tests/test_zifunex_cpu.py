"""Zifunex without a GPU: configuration, spec, tensor names, cache and state bookkeeping, the oracle's own parts."""

import json

import pytest
import torch

import plain_zifunex as plain
from tinyvllm_b200.cache.storage import CacheStorage, group_runs
from tinyvllm_b200.config.registry import ConfigError, parse_model_config
from tinyvllm_b200.engine.model import Model
from tinyvllm_b200.models import ZifunexConfig
from tinyvllm_b200.parts.base import EMBEDDING, KVNeed, StateNeed, kv_need, state_needs
from tinyvllm_b200.weights.loader import WeightsError, bind_tensors
from tinyvllm_b200.weights.random_init import random_tensors
from zifunex_configs import ZIFUNEX_CONFIGS, ZIFUNEX_DECAY_RANKS, ZIFUNEX_SEEDS, tensors_of

F64 = torch.float64


@pytest.mark.parametrize("name", sorted(ZIFUNEX_CONFIGS))
def test_config_round_trip_and_registry(name):
    config = ZIFUNEX_CONFIGS[name]
    data = json.loads(json.dumps(config.to_json()))
    assert data["architecture"] == "Zifunex"
    again = parse_model_config(data)
    assert isinstance(again, ZifunexConfig) and again == config and again.to_json() == data


def test_config_refusals():
    good = ZIFUNEX_CONFIGS["a"].to_json()
    for change in (lambda d: d.pop("norm"), lambda d: d.pop("width"), lambda d: d.pop("streams"),
                   lambda d: d.update(streams=0),
                   lambda d: d["embedding"]["bigram"].pop("mul_prev"),
                   lambda d: d["embedding"]["bigram"].update(buckets=0),
                   lambda d: d["loop"].pop("times"), lambda d: d["loop"].update(times=0),
                   lambda d: d["loop"].update(stop=5), lambda d: d["loop"].update(start=3),
                   lambda d: d["layers"][0].update(type="serial"),
                   lambda d: d["layers"][0]["mixer"].pop("right"),
                   lambda d: d["layers"][0]["mixer"]["left"].pop("vdim"),
                   lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3),
                   lambda d: d["layers"][0]["mixer"]["left"].update(softcap=0.0),
                   lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=18),
                   lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=7),
                   lambda d: d["layers"][0]["mixer"]["right"].pop("dt_rank"),
                   lambda d: d["layers"][0]["mixer"]["right"].update(conv=0),
                   lambda d: d["layers"][1]["mixer"].pop("tau"),
                   lambda d: d["layers"][1]["mixer"].update(tau=0),
                   lambda d: d["layers"][1]["mlp"].update(kind="moe"),
                   lambda d: d["layers"][1]["mlp"].pop("ff")):
        data = json.loads(json.dumps(good))
        change(data)
        with pytest.raises(ConfigError):
            parse_model_config(data)


@pytest.mark.parametrize("name", sorted(ZIFUNEX_CONFIGS))
def test_the_model_declares_exactly_the_checkpoint_tensors(name):
    config = ZIFUNEX_CONFIGS[name]
    model = Model(config.to_spec(), device="cpu", dtype=torch.float32)
    declared, shapes, free = {}, {}, set()
    for _, spec in model.param_targets():
        assert not spec.optional
        for source in spec.sources:
            declared[source.name] = declared.get(source.name, 0) + 1
            shapes[source.name] = (source.rows,) + (tuple(spec.shape[1:]) if source.cols is None else (source.cols,))
            if spec.free_rows or spec.free_cols:
                free.add(source.name)
    tensors = tensors_of(config, ZIFUNEX_SEEDS[name], ZIFUNEX_DECAY_RANKS[name])
    assert set(declared) == set(tensors)
    assert all(count == 1 for count in declared.values())
    assert all(tuple(tensors[n].shape) == shapes[n] for n in tensors if n not in free)
    # only the rank of the decays' projection is left to the checkpoint
    assert free == {f"l{i}.mix.{a}" for i, layer in enumerate(config.layers) if layer.linear is not None for a in ("a1", "a2")}
    for index, layer in enumerate(config.layers):
        assert any(n.startswith(f"l{index}.hc2") for n in tensors) == (layer.ff is not None)


@pytest.mark.parametrize("name", sorted(ZIFUNEX_CONFIGS))
def test_weights_are_bound_and_packed(name):
    """Every tensor finds its place: the packed input projections hold the mixers' rows in order, the decays' first
    step joined to them with its rank widened to a multiple of 8, the taps stand by age with zeros in front."""
    config = ZIFUNEX_CONFIGS[name]
    rank = ZIFUNEX_DECAY_RANKS[name]
    tensors = tensors_of(config, ZIFUNEX_SEEDS[name], rank)
    model = Model(config.to_spec(), device="cpu", dtype=torch.float32)
    bind_tensors(model.param_targets(), tensors, dtype=torch.float32, device="cpu")
    model._after_binding()
    for index, (layer, block) in enumerate(zip(config.layers, model.blocks)):
        at = f"l{index}.mix."
        if layer.linear is not None:
            mixer = block.mixer
            assert mixer.decay_rank == -(-rank // 8) * 8 and mixer.decay_rank >= rank
            want = torch.cat([tensors[at + n] for n in ("q", "k", "v", "g", "a1")])
            assert torch.equal(mixer.in_weight[:want.shape[0]], want) and not mixer.in_weight[want.shape[0]:].any()
            assert torch.equal(mixer.a2_weight[:, :rank], tensors[at + "a2"]) and not mixer.a2_weight[:, rank:].any()
        else:
            want = torch.cat([tensors[at + n] for n in ("left.q", "left.k", "left.v", "right.in")])
            assert torch.equal(block.mixer.in_weight, want)
            scan, taps = block.mixer.right, layer.right.conv
            assert torch.equal(scan.conv_by_tap[-taps:], tensors[at + "right.conv"].t())
            assert not scan.conv_by_tap[:-taps].any() and scan.conv_by_tap.shape[0] >= 2
            assert torch.allclose(scan.a, -torch.exp(tensors[at + "right.A_log"]))
            n, r = layer.right.state, layer.right.dt_rank
            assert torch.equal(scan.x_weight[:r], tensors[at + "right.x"][:r])
            assert torch.equal(scan.x_weight[scan.rank_cols:scan.rank_cols + 2 * n], tensors[at + "right.x"][r:])
            assert scan.x_weight.shape[0] % 8 == 0 and scan.rank_cols % 8 == 0
            assert not scan.x_weight[r:scan.rank_cols].any() and not scan.x_weight[scan.rank_cols + 2 * n:].any()
    model._after_binding()                                   # a second time changes nothing


def test_ranks_that_do_not_fit_are_refused():
    config = ZIFUNEX_CONFIGS["g"]
    tensors = tensors_of(config, 1, 7)
    tensors["l0.mix.a2"] = tensors["l0.mix.a2"][:, :6].contiguous()
    model = Model(config.to_spec(), device="cpu", dtype=torch.float32)
    bind_tensors(model.param_targets(), tensors, dtype=torch.float32, device="cpu")
    with pytest.raises(ValueError, match="a1 has 7 rows"):
        model._after_binding()
    tensors["l0.mix.a1"] = tensors["l0.mix.a1"][:, :60].contiguous()
    with pytest.raises(WeightsError, match="l0.mix.a1"):     # the width is not left to the checkpoint
        bind_tensors(Model(config.to_spec(), device="cpu", dtype=torch.float32).param_targets(), tensors,
                     dtype=torch.float32, device="cpu")


def test_random_weights_cover_every_tensor():
    model = Model(ZIFUNEX_CONFIGS["b"].to_spec(), device="cpu", dtype=torch.float32)
    targets = model.param_targets()
    bind_tensors(targets, random_tensors(targets, 3), dtype=torch.float32, device="cpu")
    model._after_binding()
    assert abs(model.blocks[0].mixer_connection.w_in.sum().item() - 1.0) < 0.3


@pytest.mark.parametrize("name", sorted(ZIFUNEX_CONFIGS))
def test_every_layer_run_has_pages_and_states_of_its_own(name):
    """A loop's passes each own their cache and states; parallel layers keep keys and values and two states beside
    them; the pair embedding keeps one token a request."""
    config = ZIFUNEX_CONFIGS[name]
    model = Model(config.to_spec(), device="cpu", dtype=torch.bfloat16)
    needs, order = model.cache_needs(), config.run_order()
    loop = config.loop
    assert len(needs) == len(order) == len(config.layers) + (0 if loop is None else (loop.stop - loop.start) * (loop.times - 1))
    for index, need in zip(order, needs):
        layer = config.layers[index]
        if layer.linear is not None:
            lin = layer.linear
            assert need == StateNeed((lin.heads, lin.dim, lin.vdim), torch.float32)
            continue
        left, right = layer.left, layer.right
        assert kv_need(need) == KVNeed(left.kv_heads, left.dim, None, left.vdim, 0)
        scan, conv = state_needs(need)
        assert scan.shape == (right.inner, right.state) and scan.dtype == torch.float32
        assert conv.shape[0] >= max(1, right.conv - 1) and conv.shape[1] == right.inner and conv.dtype == torch.float32
    groups, where = group_runs(needs, model.cache_sources())
    storage = CacheStorage(groups, where, needs, page_size=4, pages_per_group=3, num_state_slots=2, dtype=torch.float32,
                           device="cpu", other_states=model.other_states())
    states = sum(1 if config.layers[i].linear is not None else 2 for i in order)
    assert len(storage.state) == states + (config.bigram is not None)
    for run, index in enumerate(order):
        if config.layers[index].linear is None:
            assert storage.state_of(run, f"l{index}.mix.right.scan").shape[0] == 2
            assert storage.kv_of(run)[0].shape[0] == 3
    if config.bigram is not None:
        assert storage.state_of(EMBEDDING).dtype == torch.int32
    for arena in storage.state.values():
        arena.fill_(3)
    saved = storage.snapshot_state([1])
    storage.clear_state([1])
    assert all((arena[0] == 3).all() and (arena[1] == 0).all() for arena in storage.state.values())
    storage.restore_state(saved)
    assert all((arena == 3).all() for arena in storage.state.values())


def test_run_order():
    from dataclasses import replace
    from tinyvllm_b200.models.zifunex import ZifunexLoop
    config = ZIFUNEX_CONFIGS["a"]
    assert config.run_order() == (0, 1, 2, 1, 2, 3)
    assert replace(config, loop=None).run_order() == (0, 1, 2, 3)
    assert replace(config, loop=ZifunexLoop(3, 4, 4)).run_order() == (0, 1, 2, 3, 3, 3, 3)
    for loop in (None, {"start": 0, "stop": 2, "times": 3}):
        data = {"layers": [None] * 4, "loop": loop}
        want = (0, 1, 2, 3) if loop is None else (0, 1, 0, 1, 0, 1, 2, 3)
        assert tuple(plain.run_order(data)) == want


# -------------------------------------------------------------- the oracle's own parts
def test_the_oracles_pairs():
    bigram = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert plain.bigram_rows([4, 1, 9], bigram) == [10, (12 + 7) % 10, (3 + 63) % 10]
    assert plain.bigram_rows([1, 9], bigram, previous=4) == plain.bigram_rows([4, 1, 9], bigram)[1:]


def test_the_oracles_streams():
    g = torch.Generator().manual_seed(1)
    x, y = torch.randn(2, 3, 5, generator=g, dtype=F64), torch.randn(2, 5, generator=g, dtype=F64)
    mix, out = torch.randn(3, 3, generator=g, dtype=F64), torch.randn(3, generator=g, dtype=F64)
    new = plain.write_streams(x, y, mix, out)
    for t in range(3):
        want = sum(mix[s, t] * x[:, s] for s in range(3)) + out[t] * y
        assert torch.allclose(new[:, t], want)
    assert torch.allclose(plain.read_streams(x, out), sum(out[s] * x[:, s] for s in range(3)))


def test_the_oracles_norms_and_cap():
    x = torch.tensor([[3.0, 4.0, 0.0, 1.0]], dtype=F64)
    one, zero = torch.ones(4, dtype=F64), torch.zeros(4, dtype=F64)
    assert torch.allclose(plain.layer_norm(x, one, zero, 1e-5), torch.nn.functional.layer_norm(x, (4,), eps=1e-5))
    pair = plain.half_sum_of_normed(x, 2 * x, one, one, 0.0)
    assert torch.allclose(pair, x / (x * x).mean().sqrt())
    s = plain.capped_scores(x.view(1, 1, 4), x.view(1, 1, 4), 1.0, 2.0)
    assert torch.allclose(s, torch.tensor(2.0, dtype=F64) * torch.tanh(torch.tensor(13.0, dtype=F64)))


def test_the_oracles_recurrences_carry_their_states():
    """Cut in two, the convolution, the scan and the linear attention give what they give whole."""
    g = torch.Generator().manual_seed(2)
    w = {"m.in": (12, 5), "m.conv": (6, 3), "m.conv.b": (6,), "m.x": (2 + 8, 6), "m.dt": (6, 2), "m.dt.b": (6,),
         "m.A_log": (6, 4), "m.D": (6,), "m.o": (5, 6), "n.q": (6, 5), "n.k": (6, 5), "n.v": (8, 5), "n.g": (8, 5),
         "n.a1": (3, 5), "n.a2": (6, 3), "n.a2.b": (6,), "n.norm": (4,), "n.o": (5, 8)}
    w = {name: torch.randn(shape, generator=g, dtype=F64) for name, shape in w.items()}
    h = torch.randn(9, 5, generator=g, dtype=F64)
    mixer = {"inner": 6, "state": 4, "dt_rank": 2, "conv": 3}
    whole, state, tail = plain.mamba(h, w, "m", mixer)
    first, s1, t1 = plain.mamba(h[:4], w, "m", mixer)
    second, s2, t2 = plain.mamba(h[4:], w, "m", mixer, state=s1, before=t1)
    assert torch.allclose(torch.cat([first, second]), whole) and torch.allclose(s2, state) and torch.allclose(t2, tail)
    taps = torch.nn.functional.conv1d(torch.nn.functional.pad((h @ w["m.in"].T)[:, :6].T, (2, 0))[None],
                                      w["m.conv"][:, None], w["m.conv.b"], groups=6)[0].T
    assert torch.allclose(plain.causal_convolution((h @ w["m.in"].T)[:, :6], w["m.conv"], w["m.conv.b"])[0], taps)
    mixer = {"heads": 2, "dim": 3, "vdim": 4, "tau": 2.0}
    whole, state = plain.gla(h, w, "n", mixer, 1e-6)
    first, s1 = plain.gla(h[:4], w, "n", mixer, 1e-6)
    second, s2 = plain.gla(h[4:], w, "n", mixer, 1e-6, state=s1)
    assert torch.allclose(torch.cat([first, second]), whole) and torch.allclose(s2, state)
    alpha = plain.channel_decays(h, w, "n", 2.0)
    assert torch.allclose(alpha ** 2, torch.sigmoid(h @ w["n.a1"].T @ w["n.a2"].T + w["n.a2.b"]))

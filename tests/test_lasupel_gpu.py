"""Lasupel on the GPU against the plain implementation: each mechanism alone, then whole models through
the step function, the trace program and the generation entry point."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_lasupel as plain
import replay_helpers as rh
from lasupel_configs import (LASUPEL_CONFIGS, LASUPEL_PAGES, LASUPEL_SEEDS, greedy_oracle, oracle_logits, tokens_of,
                             write_folder)

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
IDS = ["f32", "bf16"]
CUDA = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write_folder(tmp_path_factory.mktemp(f"lasupel_{name}"), config, LASUPEL_SEEDS[name])
            for name, config in LASUPEL_CONFIGS.items()}


def close(got, want, dtype, scale=None, limit=None):
    scale = scale if scale is not None else max(want.abs().max().item(), 1e-6)
    limit = limit or (4e-6 if dtype == torch.float32 else 1.2e-2)
    worst = (got.double().cpu() - want.double().cpu()).abs().max().item() / scale
    assert worst <= limit, f"largest difference {worst:.3g} of the scale, allowed {limit:.3g}"


def rounded(t, dtype):
    """Values of ``t`` as ``dtype`` stores them, in float64."""
    return t.to(dtype).double()


def dev(t, kind=torch.float32):
    return t.to(kind).contiguous().to(CUDA)


def ints(values):
    return torch.tensor(values, dtype=torch.int32, device=CUDA)


def entries_of(lengths, slots, padding=()):
    """row_starts, state_slots and token_row of a step's entries; rows in ``padding`` belong to nobody."""
    starts = [0]
    for length in lengths:
        starts.append(starts[-1] + length)
    rows = [-1 if r in padding else r for r, n in enumerate(lengths) for _ in range(n)]
    return dict(row_starts=ints(starts), state_slots=ints(slots), token_row=ints(rows)), starts


# ------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width", [50, 64, 1028, 4096])
def test_scaled_embedding_starts_the_stream(width, dtype):
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(width)
    table = rounded(torch.randn(83, width, generator=g), dtype)
    ids = torch.randint(0, 83, (21,), generator=g).tolist()
    for scale in (0.3, 1.0, 45.25):
        stream, low = kernels.embed_scaled(dev(table, dtype), ints(ids), scale)
        assert stream.dtype == torch.float32 and low.dtype == dtype
        close(stream, table[ids] * scale, torch.float32, limit=1e-6)
        assert torch.equal(low, stream.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("width", [50, 64, 384, 4096])
def test_norm_behind_a_sublayer_and_the_rounded_stream(width, dtype):
    """s + y / rms(y) * w and its rounding in one pass; tiny outputs, where the eps decides; a stream that nothing is
    added to is only rounded."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(width)
    eps, tokens = 1e-4, 9
    weight = (1.0 + 0.3 * torch.randn(width, generator=g)).to(dtype)
    s = (torch.randn(tokens, width, generator=g) * 5.0).float()
    y = torch.randn(tokens, width, generator=g).float() * torch.tensor([1e-3, 1e-2, 1.0, 30.0, 1.0, 0.0, 2.0, 4.0, 1e-4])[:, None]
    want = s.double() + plain.over_rms(y.double(), eps) * weight.double()
    stream = dev(s)
    low, same = kernels.sandwich_norm(stream, dev(y), post_weight=weight.to(CUDA), post_eps=eps, out_dtype=dtype, rounded=True)
    assert same is stream and low.dtype == dtype and torch.equal(low, stream.to(dtype))
    close(stream, want, torch.float32, limit=2e-6)
    low, same = kernels.sandwich_norm(dev(s), None, out_dtype=dtype, rounded=True)
    assert torch.equal(low.cpu(), s.to(dtype)) and torch.equal(same.cpu(), s)
    nothing, same = kernels.sandwich_norm(dev(s), dev(y), post_weight=weight.to(CUDA), post_eps=eps, out_dtype=dtype)
    assert nothing is None
    close(same, want, torch.float32, limit=2e-6)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("taps,channels", [(1, 12), (2, 64), (3, 37), (4, 256), (9, 72)])
def test_convolution_of_biased_inputs(taps, channels, dtype):
    """Inputs with a bias: a fresh request starts from zeros, not from the bias; carried inputs hold it."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(taps * 100 + channels)
    kernel_taps = next(k for k in kernels.CONV_TAPS if k >= taps)
    lengths, slots = [50, 2, 1, 19, 1], [2, 4, 0, 5, 1]
    entries, starts = entries_of(lengths, slots)
    x = rounded(torch.randn(starts[-1], channels, generator=g), dtype)
    in_bias, bias = 3.0 + torch.randn(channels, generator=g).float(), torch.randn(channels, generator=g).float()
    by_tap = torch.zeros(kernel_taps, channels)
    w = torch.randn(channels, taps, generator=g)
    by_tap[kernel_taps - taps:] = w.t()
    state = torch.randn(6, kernel_taps - 1, channels, generator=g).float()
    state[[2, 0]] = 0.0                                            # two fresh requests
    device_state = dev(state)
    got = kernels.short_convolution(dev(x, dtype), dev(by_tap), bias=dev(bias), act=None, in_bias=dev(in_bias),
                                    state=device_state, **entries)
    want_state = state.double().clone()
    for r, slot in enumerate(slots):
        rows = slice(starts[r], starts[r + 1])
        y, want_state[slot] = plain.causal_convolution(x[rows] + in_bias.double(), by_tap.t().double(), state[slot].double())
        close(got[rows], y + bias.double(), dtype, scale=max(1.0, y.abs().max().item()), limit=4e-6 if dtype == torch.float32 else 6e-3)
    close(device_state, want_state, torch.float32, limit=1e-6)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("blocks,size,n,tokens", [(1, 64, 128, 5), (4, 24, 48, 70), (3, 13, 26, 9), (16, 8, 16, 130), (31, 1, 2, 66),
                                                  (1, 1600, 40, 3), (2, 256, 512, 200)])
def test_products_of_parts(blocks, size, n, tokens, dtype):
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(blocks * 100 + size)
    wide = rounded(torch.randn(tokens, blocks * size + 8, generator=g), dtype)
    w = rounded(torch.randn(blocks, n, size, generator=g), dtype)
    got = kernels.block_products(dev(wide, dtype)[:, 8:], dev(w, dtype))
    assert got.dtype == torch.float32 and got.shape == (tokens, blocks, n)
    want = torch.einsum("tbk,bnk->tbn", wide[:, 8:].reshape(tokens, blocks, size), w)
    close(got, want, torch.float32, limit=1e-5)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("blocks,size", [(1, 64), (4, 24), (3, 13), (16, 8), (31, 1), (2, 130), (2, 256)])
def test_recurrent_unit_from_a_carried_state(blocks, size, dtype):
    """Five entries from carried states, one longer than three of the scan's blocks, ends of entries on both sides of a
    block's; then steps of single tokens in numbers that share weights differently, with the gates' products inside and
    outside, beside the scan.  Channel 0 keeps nearly everything, takes token 2 in alone and must still hold it 400
    tokens later."""
    from tinyvllm_b200.ops import kernels

    channels = blocks * size
    g = torch.Generator().manual_seed(channels)
    f32 = lambda *shape, spread=1.0: (torch.randn(*shape, generator=g) * spread).float()
    lengths, slots = [403, 128, 1, 129, 2], [3, 0, 5, 1, 4]
    entries, starts = entries_of(lengths, slots)
    tokens = starts[-1]
    lam = torch.rand(channels, generator=g) * 9.0 - 8.0
    br, bi, by = f32(channels, spread=0.5), f32(channels, spread=0.5), f32(channels, spread=0.5)
    w = rounded(f32(blocks, 2 * size, size, spread=size ** -0.5), dtype)
    w[0, 0], w[0, size] = 0.0, 0.0
    lam[0], br[0], bi[0], by[0] = -9.0, 0.0, 20.0, 3.0
    u, y = rounded(f32(tokens, channels), dtype), rounded(f32(tokens, channels + 4), dtype)
    u[:403, 0], u[2, 0] = 0.0, 50.0
    ys = y[:, 3:3 + channels]
    ra, ri = w[:, :size], w[:, size:]
    state = f32(6, channels, spread=0.5)
    state[3] = 0.0
    decay = dev(-8.0 * torch.nn.functional.softplus(lam.double()))

    def reference(u, ys, state):
        r = plain.block_gate(u, ra, br.double().view(blocks, size))
        i = plain.block_gate(u, ri, bi.double().view(blocks, size))
        s, state = plain.gated_linear_unit_scan(u, r, i, lam.double(), state)
        return s * plain.gelu_tanh(ys + by.double()), s, state

    want, want_state = [], state.double().clone()
    for r, slot in enumerate(slots):
        rows = slice(starts[r], starts[r + 1])
        out, s, want_state[slot] = reference(u[rows], ys[rows], state[slot].double())
        want.append(out)
        if r == 0:
            assert s[402, 0] > 0.75 * s[2, 0] > 1.0
    want = torch.cat(want)
    common = dict(blocks=blocks, decay=decay, bias_r=dev(br), bias_i=dev(bi), bias_y=dev(by))
    du, dw = dev(u, dtype), dev(w, dtype)
    device_state = dev(state)
    out = torch.full((tokens, channels + 5), 7.0, dtype=dtype, device=CUDA)
    kernels.recurrent_unit(du, dev(y, dtype)[:, 3:3 + channels], pre=kernels.block_products(du, dw), state=device_state,
                           out=out[:, 2:2 + channels], **common, **entries)
    limit = 1e-5 if dtype == torch.float32 else None
    close(out[:, 2:2 + channels], want, dtype, limit=limit)
    close(device_state, want_state, torch.float32, limit=1e-5 if dtype == torch.float32 else 1e-4)
    assert torch.equal(device_state[2].cpu(), state[2]) and (out[:, :2] == 7.0).all() and (out[:, 2 + channels:] == 7.0).all()
    for count, padding in ((1, ()), (2, ()), (3, (1,)), (7, (3,)), (13, (12,)), (21, (20,))):
        all_slots = torch.randperm(count + 2, generator=g)[:count].tolist()
        entries, _ = entries_of([1] * count, all_slots, padding)
        state = f32(count + 2, channels, spread=0.5)
        want_state = state.double().clone()
        inside, outside, scanned = dev(state), dev(state), dev(state)
        for _ in range(3):
            u, ys = rounded(f32(count, channels), dtype), rounded(f32(count, channels), dtype)
            want = torch.zeros(count, channels, dtype=F64)
            for r, slot in enumerate(all_slots):
                if r not in padding:
                    want[r:r + 1], _, want_state[slot] = reference(u[r:r + 1], ys[r:r + 1], want_state[slot])
            du, dy = dev(u, dtype), dev(ys, dtype)
            pre = kernels.block_products(du, dw)
            for device_state, more in ((inside, dict(weight=dw, single=True)), (outside, dict(pre=pre, single=True)),
                                       (scanned, dict(pre=pre))):
                got = kernels.recurrent_unit(du, dy, state=device_state, **more, **common, **entries)
                close(got, want, dtype, limit=limit)
                close(device_state, want_state, torch.float32, limit=1e-5 if dtype == torch.float32 else 1e-4)
                assert (got[list(padding)] == 0).all()
        untouched = [s for s in range(count + 2) if s not in all_slots] + [all_slots[p] for p in padding]
        assert torch.equal(inside[untouched].cpu(), state[untouched])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_slow_channels_do_not_drift(dtype):
    """Channels that lose a thousandth to a ten-thousandth a token over 6,000 tokens: an exponential that is one unit off
    to one side would be off by hundreds of units at the end.  So for heads of the delta rule that lose as little."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(3)
    tokens, channels = 6000, 64
    entries, _ = entries_of([tokens], [0])
    lam = torch.linspace(-10.0, -6.5, channels).float()
    u, pre = torch.ones(tokens, channels), torch.zeros(tokens, 2, channels)
    pre[:, 0] = torch.randn(tokens, channels, generator=g) * 0.3
    zero = torch.zeros(channels)
    decay = -8.0 * torch.nn.functional.softplus(lam.double())
    state = torch.zeros(1, channels, device=CUDA)
    kernels.recurrent_unit(dev(u, dtype), dev(u, dtype), blocks=1, decay=dev(decay), bias_r=dev(zero), bias_i=dev(zero),
                           pre=dev(pre.view(tokens, 1, 2 * channels)), state=state, act=None, **entries)
    log_a = decay.float().double() * torch.sigmoid(pre[:, 0].double())
    assert log_a.mean(0).max() > -3e-4 and log_a.mean(0).min() < -3e-3
    later = log_a.flip(0).cumsum(0).flip(0) - log_a                # the decays behind each token
    want = (torch.exp(later) * torch.sqrt(-torch.expm1(2.0 * log_a)) * 0.5).sum(0)
    close(state[0] / want.float().to(CUDA), torch.ones(channels), torch.float32, limit=2e-5 if dtype == torch.float32 else 6e-5)
    heads, dim = 4, 8
    rate = -torch.tensor([1e-4, 3e-4, 1e-3, 3e-3])
    mixed, proj = torch.ones(tokens, 3 * heads * dim), torch.zeros(tokens, 2 * heads)
    proj[:, :heads], proj[0, :heads] = -200.0, 200.0               # the first token alone writes
    proj[:, heads:] = torch.rand(tokens, heads, generator=g)
    proj = rounded(proj, dtype)
    state = torch.zeros(1, heads, dim, dim, device=CUDA)
    kernels.delta_rule(dev(mixed, dtype), dev(proj, dtype), q_at=0, k_at=heads * dim, v_at=2 * heads * dim, beta_at=0,
                       decay_at=heads, heads=heads, key_heads=heads, dim=dim, vdim=dim, rate=dev(rate), dt_bias=dev(torch.zeros(heads)),
                       state=state, raw_out=torch.empty(tokens, heads * dim, device=CUDA), **entries)
    kept = torch.exp((rate.double() * plain.softplus(proj[1:, heads:])).sum(0)) / (dim + 1e-6) ** 0.5
    close(state[0].cpu().double() / kept[:, None, None], torch.ones(heads, dim, dim), torch.float32, limit=2e-5)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 16, 32), (3, 1, 10, 7), (2, 2, 32, 48), (1, 1, 5, 3), (4, 2, 64, 128),
                                               (4, 1, 130, 24), (2, 1, 128, 128), (2, 1, 256, 40), (2, 2, 33, 256)])
def test_delta_rule_from_a_carried_state(heads, kv, dim, vdim, dtype):
    """Five entries from carried states (ends on both sides of the scan's blocks), then single tokens in the one-launch
    form beside a padding row and beside the scan.  In the first entry head 0 decays by nothing and writes token 2 alone;
    the query 400 tokens later asks for its key and must find its value.  In the second entry every token has one key and
    writes fully: what is read is the newest value."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(heads * 1000 + dim)
    per, hv = kv * dim, heads * vdim
    q_at, k_at, v_at = 1, 2 + per, 3 + 2 * per
    beta_at, decay_at, gate_at = 2, 3 + heads, 5 + 2 * heads
    scale, unit_eps, eps = dim ** -0.5, 1e-6, 1e-5
    a_log = torch.linspace(-5.0, 1.0, heads).float()
    dt_bias = torch.randn(heads, generator=g).float() * 0.5
    weight = (1.0 + 0.2 * torch.randn(vdim, generator=g)).float()
    shared = [h // (heads // kv) for h in range(heads)]

    def project(count):
        mixed = rounded(torch.randn(count, v_at + hv + 2, generator=g), dtype)
        proj = rounded(torch.randn(count, gate_at + hv, generator=g), dtype)
        return mixed, proj

    def reference(mixed, proj, state):
        q = plain.unit(mixed[:, q_at:q_at + per].reshape(-1, kv, dim))[:, shared] * scale
        k = plain.unit(mixed[:, k_at:k_at + per].reshape(-1, kv, dim))[:, shared]
        v = mixed[:, v_at:v_at + hv].reshape(-1, heads, vdim)
        beta = torch.sigmoid(proj[:, beta_at:beta_at + heads])
        decay = torch.exp(-torch.exp(a_log.double()) * plain.softplus(proj[:, decay_at:decay_at + heads] + dt_bias.double()))
        o, state = plain.delta_rule(q, k, v, decay, beta, state)
        out = (plain.over_rms(o, eps) * weight.double()).reshape(-1, hv) * plain.silu(proj[:, gate_at:gate_at + hv])
        return out, o.reshape(-1, hv), state

    lengths, slots = [403, 40, 1, 9, 2], [3, 0, 5, 1, 4]
    entries, starts = entries_of(lengths, slots)
    mixed, proj = project(starts[-1])
    proj[:403, beta_at], proj[2, beta_at], proj[:403, decay_at] = -60.0, 30.0, -60.0
    mixed[402, q_at:q_at + dim] = mixed[2, k_at:k_at + dim]
    mixed[403:443, k_at:k_at + per] = mixed[403, k_at:k_at + per]
    mixed[403:443, q_at:q_at + per] = mixed[403, k_at:k_at + per]
    proj[403:443, beta_at:beta_at + heads] = 30.0
    state = (torch.randn(6, heads, dim, vdim, generator=g) * 0.3).float()
    state[3] = 0.0
    want, raw, want_state = [], [], state.double().clone()
    for r, slot in enumerate(slots):
        out, o, want_state[slot] = reference(mixed[starts[r]:starts[r + 1]], proj[starts[r]:starts[r + 1]], state[slot].double())
        want.append(out)
        raw.append(o)
    assert torch.allclose(raw[0][402, :vdim] / scale, mixed[2, v_at:v_at + vdim], atol=1e-3)
    assert torch.allclose(raw[1] / scale, mixed[403:443, v_at:v_at + hv], atol=1e-3)
    want, raw = torch.cat(want), torch.cat(raw)
    common = dict(q_at=q_at, k_at=k_at, v_at=v_at, beta_at=beta_at, decay_at=decay_at, gate_at=gate_at, heads=heads,
                  key_heads=kv, dim=dim, vdim=vdim, rate=dev(-torch.exp(a_log)), dt_bias=dev(dt_bias), query_scale=scale,
                  unit_eps=unit_eps, norm_weight=dev(weight), eps=eps)
    # a norm over a head multiplies what cancelled in the head's sum: the bound is on the scale of all heads
    limit = 1e-4 if dtype == torch.float32 else None
    for cols in (0, 2, 4):
        device_state = dev(state)
        device_raw = torch.empty(starts[-1], hv, device=CUDA)
        got = kernels.delta_rule(dev(mixed, dtype), dev(proj, dtype), state=device_state, raw_out=device_raw, cols=cols,
                                 **common, **entries)
        # inputs are exact in both number formats, and all that follows them but the last rounding is float32
        close(device_raw, raw, torch.float32, limit=1e-5)
        close(device_state, want_state, torch.float32, limit=1e-5)
        close(got, want, dtype, limit=limit)
        assert torch.equal(device_state[2].cpu(), state[2])
    slots = [5, 2, 7, 0, 6, 1, 3]
    entries, _ = entries_of([1] * 7, slots, padding=(3,))
    state = (torch.randn(8, heads, dim, vdim, generator=g) * 0.5).float()
    step_state, scan_state, want_state = dev(state), dev(state), state.double().clone()
    for _ in range(3):
        mixed, proj = project(7)
        want = torch.zeros(7, hv, dtype=F64)
        for r in range(7):
            if r != 3:
                want[r:r + 1], _, want_state[slots[r]] = reference(mixed[r:r + 1], proj[r:r + 1], want_state[slots[r]])
        for device_state, more in ((step_state, {}), (scan_state, dict(raw_out=torch.empty(7, hv, device=CUDA)))):
            got = kernels.delta_rule(dev(mixed, dtype), dev(proj, dtype), state=device_state, **more, **common, **entries)
            close(got, want, dtype, limit=limit)
            close(device_state, want_state, torch.float32, limit=1e-5)
            assert (got[3] == 0).all()
    assert torch.equal(step_state[[4, 0]].cpu(), state[[4, 0]])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("experts,top,groups,keep,ff,limit", [(8, 3, 2, 1, 24, 1.0), (6, 2, 3, 2, 10, 0.3), (5, 5, 1, 1, 16, 50.0),
                                                              (64, 8, 8, 3, 32, 2.0), (4, 1, 4, 1, 7, 1.0), (200, 4, 40, 1, 8, 0.7)])
@pytest.mark.parametrize("tokens", [3, 400])
def test_softmax_routing_with_groups_and_clipped_experts(tokens, experts, top, groups, keep, ff, limit, dtype):
    """The chosen experts' weights are the softmax scores as they are, exactly 0 elsewhere; the first token's best group
    by its largest score is not its best by the sum of two; activations on both sides of the limits."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(experts * 10 + tokens)
    logits = (torch.randn(tokens, experts, generator=g) * 2.0).float()
    if groups > 1 and experts // groups > 1:
        size = experts // groups
        logits[0] = -3.0 + 0.01 * torch.randn(experts, generator=g)
        logits[0, :size] = 2.0 + 0.01 * torch.randn(size, generator=g)     # a group of good experts ...
        logits[0, size] = 2.5                                      # ... and one with the best
    proj = rounded(torch.randn(tokens, 2 * experts * ff, generator=g) * limit * 1.5, dtype)
    weights = plain.chosen_weights(logits.double(), top, None if groups == 1 else {"count": groups, "keep": keep})
    both = proj.view(tokens, experts, 2, ff)
    gate, up = both[:, :, 0].clamp(max=limit), both[:, :, 1].clamp(-limit, limit)
    want = (gate * torch.sigmoid(1.702 * gate) * (up + 1.0) * weights[..., None]).view(tokens, -1)
    assert (both[:, :, 0] > limit).any() or limit > 10
    got_weights = torch.empty(tokens, experts, device=CUDA)
    got, passed = kernels.route_softmax_gated(dev(logits), dev(proj, dtype), experts=experts, identity=0, top=top, ff=ff,
                                              groups=groups, keep=keep, limit=limit, alpha=1.702, weights_out=got_weights)
    assert passed is None
    close(got_weights, weights, torch.float32, limit=2e-6)
    assert torch.equal(got_weights.cpu() > 0, weights > 0)
    close(got, want, dtype, limit=4e-6 if dtype == torch.float32 else 5e-3)
    assert (got.cpu().view(tokens, experts, ff)[weights == 0] == 0).all()


# ------------------------------------------------------ attention over its own and another layer's cache
# (the reader's window, page size): windows narrower and wider than the owner's 40, inside a page, over several, all keys
READERS = [(None, 16), (75, 16), (40, 8), (17, 4), (1, 4), (130, 32)]
OWNER_WINDOW = 40


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,kv,dim,vdim,rot", [(4, 2, 32, 48, 8), (3, 1, 9, 5, 4), (8, 2, 64, 64, 64), (2, 2, 128, 32, 16)])
@pytest.mark.parametrize("window,page", READERS)
@pytest.mark.parametrize("cut", ["whole", "tail", "portions"])
def test_windows_sinks_and_a_shared_cache(cut, window, page, heads, kv, dim, vdim, rot, dtype):
    """Two attention layers run through the step function on given projections: the first writes the cache, the second
    reads it through a window of its own.  Some keys stand out for some queries, just inside and just outside both
    windows, far back and at page borders; some queries like no key at all, so that the softmax's extra term takes
    nearly everything."""
    from tinyvllm_b200.engine.model import Model
    from tinyvllm_b200.engine.step import StepRunner
    from tinyvllm_b200.models import LasupelConfig
    from tinyvllm_b200.models.lasupel import LasupelAttention, LasupelLayer
    from tinyvllm_b200.ops import attention as attention_ops

    tokens, scale = 210, 0.9 / dim ** 0.5
    rotation = {"rot_dims": rot, "rot_base": 30.0}
    sizes = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, **rotation)
    config = LasupelConfig(vocab=19, width=16, norm_eps=1e-5, layers=(
        LasupelLayer(LasupelAttention(window=OWNER_WINDOW, **sizes)),
        LasupelLayer(LasupelAttention(window=window, kv_from=0, **sizes))))
    g = torch.Generator().manual_seed(heads * 100 + dim)
    q = [torch.randn(tokens, heads, dim, generator=g) for _ in range(2)]
    k, v = torch.randn(tokens, kv, dim, generator=g), torch.randn(tokens, kv, vdim, generator=g)
    # standing out: the turned parts of both are small, the rest lies along one axis
    rest = dim - rot
    if rest >= 2:
        def aim(query, key, layer, axis):
            k[key, 0] = 0.01 * torch.randn(dim, generator=g)
            k[key, 0, rot + axis % rest] = 4.0
            q[layer][query, 0] = 0.01 * torch.randn(dim, generator=g)
            q[layer][query, 0, rot + axis % rest] = 4.0
        axis = 0
        for layer, size in ((0, OWNER_WINDOW), (1, window or 209)):
            for query in (205, 160, 131):
                for apart in (size - 1, size):                     # the last key inside, the first outside
                    if 0 <= query + layer - apart:
                        aim(query + layer + 2 * (apart == size), query + layer + 2 * (apart == size) - apart, layer, axis)
                        axis += 1
        aim(100, page * (99 // page), 0, axis)                     # first of a page
        aim(101, page * (100 // page) - 1, 1, axis + 1)            # last of a page
        against = [0] + list(range(72 - OWNER_WINDOW, 72))         # queries 71 and 0 turn away from every key they see
        k[against, 0, rot + rest - 1] = k[against, 0, rot + rest - 1].abs() + 12.0
        for layer, query in ((0, 71), (0, 0), (1, 0)):
            q[layer][query, 0] = 0.0
            q[layer][query, 0, rot + rest - 1] = -4.0
    given = [torch.cat([rounded(t, dtype).reshape(tokens, -1) for t in parts], 1).to(dtype).to(CUDA)
             for parts in ((q[0], k, v), (q[1],))]
    q, k, v = [rounded(t, dtype) for t in q], rounded(k, dtype), rounded(v, dtype)
    positions = torch.arange(tokens)
    turn = {"dims": rot, "base": 30.0}
    keys = plain.over_rms(plain.rotate_halves(k, positions, turn), 1e-5)
    want = []
    for layer, size in ((0, OWNER_WINDOW), (1, window)):
        queries = plain.over_rms(plain.rotate_halves(q[layer], positions, turn), 1e-5)
        if layer == 0:
            queries_at_71 = queries[71]
        want.append(plain.attend(queries, keys, v, scale, plain.visible(positions, positions, size)).reshape(tokens, -1))

    model = Model(config.to_spec(), device=CUDA, dtype=dtype).init_random(1)
    got = [torch.full((tokens, heads * vdim), float("nan"), dtype=dtype, device=CUDA) for _ in range(2)]

    def forward_of(layer, mixer):
        def forward(x, ctx, run):
            at = ctx.positions.long()
            out = torch.empty((x.shape[0], mixer.out_cols), dtype=dtype, device=CUDA)
            attention_ops.windowed_attention(ctx, mixer, given[layer].index_select(0, at).contiguous(), 0, run, out)
            got[layer][at] = out
            return torch.zeros((x.shape[0], config.width), dtype=torch.float32, device=CUDA)
        return forward
    for layer, block in enumerate(model.blocks):
        block.mixer.forward = forward_of(layer, block.mixer)
    pages = -(-tokens // page) + 1
    runner = StepRunner(model, page_size=page, num_pages=pages, max_requests=1, max_model_len=pages * page)
    ids = {"r": [p % 19 for p in range(tokens)]}
    steps = {"whole": lambda: rh.whole(ids), "tail": lambda: rh.tail_by_one(ids, 90),
             "portions": lambda: rh.portions(ids, 5, sizes=(2, 3, 5, 8, 31, 64))}[cut]()
    with torch.inference_mode():
        rh.run_steps(runner, steps)
    for layer in range(2):
        assert torch.isfinite(got[layer].float()).all()
        close(got[layer], want[layer], dtype, limit=3e-5 if dtype == torch.float32 else 2e-2)
    if rest >= 2:
        bare = torch.softmax(torch.einsum("hd,jd->hj", queries_at_71[:1], keys[72 - OWNER_WINDOW:72, 0]) * scale, -1)
        without = (bare @ v[72 - OWNER_WINDOW:72, 0])[0]
        assert want[0][71, :vdim].norm() < 0.8 * without.norm()    # the extra term took much of it ...
        assert want[1][0, :vdim].norm() < 0.2 * v[0, 0].norm()     # ... and nearly all of it
    # pages were kept for the wider of the two windows, and no longer
    kept = max(OWNER_WINDOW, window) if window is not None else tokens
    assert runner.manager.groups[0].window == (None if window is None else kept)


# ---------------------------------------------------------------- whole models
def requests_of(name):
    vocab = LASUPEL_CONFIGS[name].vocab
    return {f"{name}{n}": tokens_of(vocab, n, 500 + n) for n in (1, 2, 37, 150, 420)}


def make_runner(folder, dtype, page, pages, max_len=None, max_requests=4):
    from tinyvllm_b200 import read_model_config
    from tinyvllm_b200.engine.model import Model
    from tinyvllm_b200.engine.step import StepRunner

    model = Model(read_model_config(folder).to_spec(), device=CUDA, dtype=dtype).load(folder)
    return StepRunner(model, page_size=page, num_pages=pages, max_requests=max_requests,
                      max_model_len=max_len or pages * page)


def compare(got: dict, folder, requests, dtype):
    """float32: every row within rounding of the plain logits.  bfloat16: the median row and nine rows in ten within
    the rounding of 16-bit activations.  The others are tokens whose choice of experts is a close call, which 16-bit
    activations may decide otherwise, and tokens whose read-out of the delta rule nearly cancels, whose norm over a head
    then makes rounding a direction."""
    expected = oracle_logits(folder, requests)
    assert got, "no logits came back"
    errors = []
    for (rid, position), row in got.items():
        want = expected[rid]
        assert torch.isfinite(row).all()
        errors.append(((row.double() - want[position].double()).abs().max().item() / want.abs().max().item(), rid, position))
    errors.sort()
    worst, median, most = errors[-1], errors[len(errors) // 2][0], errors[len(errors) * 9 // 10][0]
    if dtype == torch.float32:
        assert worst[0] <= 5e-5, f"largest difference {worst[0]:.3g} of the largest logit, at {worst[1:]}"
    else:
        assert median <= 2e-2 and most <= 6e-2, \
            f"median {median:.3g}, ninth decile {most:.3g} of the largest logit, worst {worst}"


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", sorted(LASUPEL_CONFIGS))
@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed"])
def test_every_way_of_cutting_gives_the_plain_logits(cut, name, dtype, folders):
    """Whole prompts; prompts whose last 40 tokens come one by one; portions of changing size down to two tokens, cut
    inside pages, windows, convolutions and blocks of the scans; up to four live requests with portions beside single
    tokens, in a pool with room for little more than the live tokens and four state slots, so that pages and slots that
    finished requests gave back are taken again."""
    requests = requests_of(name)
    page = LASUPEL_PAGES[name]
    steps = {"whole": lambda: rh.whole(requests), "tail": lambda: rh.tail_by_one(requests, 40),
             "portions": lambda: rh.portions(requests, 3, sizes=(2, 3, 5, 8, 13, 31, 64, 100, 200)),
             "mixed": lambda: rh.mixed(requests, 4, live=4, decode_tail=20, sizes=(2, 3, 7, 16, 40, 90))}[cut]()
    pages = -(-rh.live_token_need(steps, page) // page) if cut == "mixed" else max(64, -(-448 // page))
    runner = make_runner(folders[name], dtype, page, pages)
    with torch.inference_mode():
        got = rh.run_steps(runner, steps)
    compare(got, folders[name], requests, dtype)
    assert not runner.manager.open_requests()
    assert all(runner.manager.free_pages(g) == pages for g in range(len(runner.manager.groups)))


@pytest.mark.parametrize("name", sorted(LASUPEL_CONFIGS))
def test_the_stream_after_every_layer(name, folders):
    """float32: the residual stream after each layer (what is pending on it added) against the plain implementation."""
    from lasupel_configs import read_folder

    tokens = tokens_of(LASUPEL_CONFIGS[name].vocab, 60, 77)
    config, tensors = read_folder(folders[name])
    want: list = []
    plain.forward(config, tensors, tokens, layers_out=want)
    runner = make_runner(folders[name], torch.float32, LASUPEL_PAGES[name], 64)
    got = []
    for block in runner.model.blocks:
        def forward(hidden, residual, ctx, run, _forward=block.forward, _norm=block.mixer_norm):
            out = _forward(hidden, residual, ctx, run)
            _, stream = _norm.settle(out[1])
            got.append(stream.clone())
            return None, stream
        block.forward = forward
    with torch.inference_mode():
        rh.run_steps(runner, rh.whole({"r": tokens}))
    assert len(got) == len(want)
    for layer, (a, b) in enumerate(zip(got, want)):
        close(a, b, torch.float32, limit=1e-5)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_a_request_is_not_moved_by_its_neighbours(dtype, folders):
    """The same request alone and beside three others, in other pages and another state slot: equal beyond
    rounding."""
    name = "e"
    requests = requests_of(name)
    page = LASUPEL_PAGES[name]
    alone = {"x": requests["e150"]}
    with torch.inference_mode():
        first = rh.run_steps(make_runner(folders[name], dtype, page, 64), rh.portions(alone, 9, sizes=(7, 50)))
        crowd = dict(list(requests.items())[2:])
        crowd["x"] = requests["e150"]
        second = rh.run_steps(make_runner(folders[name], dtype, page, 96), rh.mixed(crowd, 1, live=4, decode_tail=5))
    scale = oracle_logits(folders[name], alone)["x"].abs().max().item()
    errors = sorted((first[key].double() - second[key].double()).abs().max().item() / scale for key in first)
    if dtype == torch.float32:
        assert errors[-1] <= 2e-5
    else:                                # 16-bit rounding may settle a close choice of experts differently
        assert errors[len(errors) // 2] <= 1e-2 and errors[len(errors) * 9 // 10] <= 4e-2


def test_a_slot_that_is_taken_again_starts_from_zero(folders):
    """One state slot and pages for one request: the second request gets the slot and the pages the first
    one left, and its logits are those of a request that runs alone in a fresh pool."""
    name = "d"
    vocab = LASUPEL_CONFIGS[name].vocab
    requests = {"one": tokens_of(vocab, 50, 1), "two": tokens_of(vocab, 45, 2)}
    runner = make_runner(folders[name], torch.float32, 4, 13, max_len=52, max_requests=1)
    with torch.inference_mode():
        got = rh.run_steps(runner, rh.portions(requests, 6, sizes=(2, 11, 30)))
    compare(got, folders[name], requests, torch.float32)


@pytest.mark.parametrize("name", ["a", "b", "c", "f"])
def test_long_decoding(name, folders):
    """A prompt of five tokens and 330 tokens decoded one by one, float32: states and convolutions run along 335 tokens,
    windows pass over decoded tokens."""
    tokens = tokens_of(LASUPEL_CONFIGS[name].vocab, 335, 9)
    requests = {"long": tokens}
    page = LASUPEL_PAGES[name]
    runner = make_runner(folders[name], torch.float32, page, 352 // page, max_len=352)
    with torch.inference_mode():
        got = rh.run_steps(runner, rh.tail_by_one(requests, 330))
    compare(got, folders[name], requests, torch.float32)


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_trace_program(dtype_name, folders, tmp_path):
    name = "a"
    requests = requests_of(name)
    steps = rh.mixed(requests, 2, live=3)
    need = rh.live_token_need(steps)
    lines = "\n".join(json.dumps(step) for step in steps) + "\n"
    out = tmp_path / "out"
    root = Path(__file__).resolve().parent.parent
    done = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(folders[name]),
                           "--dtype", dtype_name, "--out", str(out), "--max-tokens", str(need)],
                          input=lines, capture_output=True, text=True, timeout=600)
    assert done.returncode == 0, done.stderr[-2000:]
    assert [line for line in done.stdout.splitlines() if line.startswith("done ")] == [f"done {s['step']}" for s in steps]
    got = rh.read_trace_output(steps, out, LASUPEL_CONFIGS[name].vocab)
    compare(got, folders[name], requests, getattr(torch, dtype_name))


@pytest.mark.parametrize("eager", [True, False], ids=["eager", "graphs"])
@pytest.mark.parametrize("name", sorted(LASUPEL_CONFIGS))
def test_greedy_generation_through_the_engine(name, eager, folders):
    """LLM.generate (scheduler, chunked prefill, decode graphs and runs of decode steps) against greedy
    decoding with the plain implementation, float32."""
    from tinyvllm_b200 import LLM, EngineConfig, SamplingParams

    config = LASUPEL_CONFIGS[name]
    prompts = [tokens_of(config.vocab, n, 700 + n) for n in (1, 9, 40, 77, 130)]
    engine_config = EngineConfig(
        model=folders[name], dtype="float32", max_model_len=512, max_num_seqs=4, max_num_batched_tokens=64,
        prefill_chunk_size=24, kv_block_size=LASUPEL_PAGES[name], kv_cache_memory_bytes=16 * 1024 * 1024,
        prefill_reserve_tokens=0, prefill_reserve_requests=0, enforce_eager=eager)
    with LLM(engine_config) as llm:
        outputs = llm.generate(prompts, SamplingParams(max_new_tokens=16, ignore_eos=True))
        if not eager:
            assert llm.engine.graph_steps > 0
    for prompt, output in zip(prompts, outputs):
        assert list(output.output_token_ids) == greedy_oracle(folders[name], prompt, 16)


def test_steps_whose_shape_comes_back_replay_from_the_right_state(folders):
    """Prompts cut into equal portions: from their third occurrence on the steps are captured and replayed; a step that
    is run a second time to be captured starts from the states it started from."""
    from tinyvllm_b200 import LLM, EngineConfig, SamplingParams

    name = "a"
    config = LASUPEL_CONFIGS[name]
    prompts = [tokens_of(config.vocab, 96, 900 + n) for n in range(6)]
    engine_config = EngineConfig(
        model=folders[name], dtype="float32", max_model_len=256, max_num_seqs=1, max_num_batched_tokens=64,
        prefill_chunk_size=24, kv_block_size=16, kv_cache_memory_bytes=16 * 1024 * 1024,
        prefill_reserve_tokens=0, prefill_reserve_requests=0)
    with LLM(engine_config) as llm:
        outputs = llm.generate(prompts, SamplingParams(max_new_tokens=3, ignore_eos=True))
        assert llm.engine.runner._step_graphs                       # some step was captured
    for prompt, output in zip(prompts, outputs):
        assert list(output.output_token_ids) == greedy_oracle(folders[name], prompt, 3)


def test_bfloat16_generation_through_the_engine(folders):
    from tinyvllm_b200 import LLM, EngineConfig, SamplingParams

    name = "e"
    config = LASUPEL_CONFIGS[name]
    prompts = [tokens_of(config.vocab, n, 800 + n) for n in (70, 3)]
    engine_config = EngineConfig(
        model=folders[name], dtype="bfloat16", max_model_len=256, max_num_seqs=4, max_num_batched_tokens=64,
        prefill_chunk_size=32, kv_block_size=16, kv_cache_memory_bytes=8 * 1024 * 1024,
        prefill_reserve_tokens=0, prefill_reserve_requests=0)
    with LLM(engine_config) as llm:
        outputs = llm.generate(prompts, SamplingParams(max_new_tokens=12, ignore_eos=True))
    assert all(len(output.output_token_ids) == 12 for output in outputs)
    for prompt, output in zip(prompts, outputs):
        logits = oracle_logits(folders[name], {"g": prompt})["g"][-1]
        top = logits.topk(2).values
        if (top[0] - top[1]).item() > 0.1 * logits.abs().max().item():
            assert output.output_token_ids[0] == int(logits.argmax())


def test_bfloat16_steps_run_on_the_tensor_core_and_one_launch_kernels(folders, monkeypatch):
    """Head sizes in steps of 16: prompt portions go to the tile kernel, decoded tokens to the kernel for single tokens,
    none to the row kernel, all with the extra term and each layer's own window; the layer that reads another's cache
    prepares queries only; decoded tokens move both recurrences' states in one launch."""
    from tinyvllm_b200.ops import kernels

    seen = {"attention_tiles": [], "attention_tiles_singles": [], "attention_rows": [], "qkv_prepare": [],
            "recurrent_unit": [], "delta_rule": []}
    for fn in seen:
        original = getattr(kernels, fn)

        def watched(*args, _original=original, _fn=fn, **kwargs):
            if "attention" in _fn:
                assert kwargs["sinks"] is not None and not kwargs["sinks"].any()
                seen[_fn].append(kwargs["window"])
            elif _fn == "qkv_prepare":
                seen[_fn].append(kwargs["num_kv"])
            else:
                seen[_fn].append(kwargs.get("weight") is not None if _fn == "recurrent_unit" else args[0].shape[0])
            return _original(*args, **kwargs)
        monkeypatch.setattr(kernels, fn, watched)
    name = "e"
    requests = {"t": tokens_of(LASUPEL_CONFIGS[name].vocab, 90, 31)}
    runner = make_runner(folders[name], torch.bfloat16, 16, 16)
    with torch.inference_mode():
        rh.run_steps(runner, rh.tail_by_one(requests, 3))
    assert seen["attention_tiles"] == [100, 60]                  # one prompt step
    assert seen["attention_tiles_singles"] == [100, 60] * 3      # three decoded tokens
    assert not seen["attention_rows"]
    assert seen["qkv_prepare"] == [2, 0] * 4
    assert seen["recurrent_unit"] == [False] + [True] * 3
    assert seen["delta_rule"] == [87, 1, 1, 1]


def test_command_line(folders, capsys):
    """python -m tinyvllm_b200 on a Lasupel folder: greedy tokens of the plain implementation, also
    streamed, and with weights drawn from a seed instead of the file."""
    from tinyvllm_b200.__main__ import main

    name = "b"
    prompts = [tokens_of(LASUPEL_CONFIGS[name].vocab, n, 950 + n) for n in (3, 45)]
    want = [greedy_oracle(folders[name], prompt, 10) for prompt in prompts]
    common = ["--model", str(folders[name]), "--max-new-tokens", "10", "--ignore-eos", "--kv-cache-mib", "16",
              "--max-model-len", "256", "--kv-block-size", "8"]
    ids = [arg for prompt in prompts for arg in ("--prompt-ids", ",".join(map(str, prompt)))]
    main(common + ["--dtype", "float32", "--stream"] + ids)
    lines = [json.loads(line) for line in capsys.readouterr().out.strip().splitlines()]
    streamed = {0: [], 1: []}
    for line in lines[:-1]:
        streamed[line["prompt"]].append(line["token_id"])
    assert [streamed[0], streamed[1]] == want
    assert [record["output_token_ids"] for record in lines[-1]["outputs"]] == want
    main(common + ["--dtype", "bfloat16", "--random-weights", "7"] + ids)
    records = json.loads(capsys.readouterr().out.strip().splitlines()[-1])["outputs"]
    assert [len(record["output_token_ids"]) for record in records] == [10, 10]

"""Zifunex on the GPU against the plain implementation: each mechanism alone, then whole models through
the step function, the trace program and the generation entry point."""

import json
import random
import subprocess
import sys
from pathlib import Path
from types import SimpleNamespace

import pytest
import torch

import plain_zifunex as plain
import replay_helpers as rh
from zifunex_configs import (ZIFUNEX_CONFIGS, ZIFUNEX_DECAY_RANKS, ZIFUNEX_PAGES, ZIFUNEX_SEEDS, greedy_oracle,
                             oracle_logits, tokens_of, write_folder)

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
IDS = ["f32", "bf16"]
CUDA = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: write_folder(tmp_path_factory.mktemp(f"zifunex_{name}"), config, ZIFUNEX_SEEDS[name],
                               ZIFUNEX_DECAY_RANKS[name])
            for name, config in ZIFUNEX_CONFIGS.items()}


def close(got, want, dtype, scale=None, limit=None):
    scale = scale if scale is not None else max(want.abs().max().item(), 1e-6)
    limit = limit or (4e-6 if dtype == torch.float32 else 1.2e-2)
    worst = (got.double().cpu() - want.double().cpu()).abs().max().item() / scale
    assert worst <= limit, f"largest difference {worst:.3g} of the scale, allowed {limit:.3g}"


def rounded(t, dtype):
    """Values of ``t`` as ``dtype`` stores them, in float64."""
    return t.to(dtype).double()


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
@pytest.mark.parametrize("width,buckets", [(64, 101), (50, 7), (1028, 1), (4096, 65521)])
def test_pair_embedding_carries_the_token_before(width, buckets, dtype):
    """Portions, single tokens and a padding row in one step; the state holds every request's last token afterwards,
    the first token of a request reads the last row whatever the state says, products beyond 32 bits wrap nowhere."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(width)
    vocab = 83
    bigram = {"buckets": buckets, "mul_prev": 2_000_000_011, "mul_cur": 1_999_999_973}
    table = rounded(torch.randn(vocab, width, generator=g), dtype)
    pairs = rounded(torch.randn(buckets + 1, width, generator=g), dtype)
    lengths, begins, slots = [40, 7, 1, 1, 2, 1], [0, 13, 0, 90, 3, 5], [2, 0, 5, 1, 4, 3]
    entries, starts = entries_of(lengths, slots, padding=(5,))
    tokens = torch.randint(0, vocab, (starts[-1],), generator=g).tolist()
    before = torch.randint(0, vocab, (6, 1), generator=g).to(torch.int32)
    state = before.to(CUDA)
    positions = [b + i for b, n in zip(begins, lengths) for i in range(n)]
    got = kernels.embed_pairs(table.to(dtype).to(CUDA), ints(tokens), positions=ints(positions), **entries,
                              pairs=dict(table=pairs.to(dtype).to(CUDA), state=state, mul_prev=bigram["mul_prev"],
                                         mul_cur=bigram["mul_cur"]))
    assert got.dtype == torch.float32
    for r, (length, begin, slot) in enumerate(zip(lengths, begins, slots)):
        mine = tokens[starts[r]:starts[r + 1]]
        if r == 5:
            close(got[starts[r]:starts[r + 1]], table[mine], torch.float32, limit=1e-6)
            assert state[slot].item() == before[slot].item()
            continue
        want = plain.embed(mine, {"embed": table, "bigram": pairs}, bigram, None if begin == 0 else before[slot].item())
        close(got[starts[r]:starts[r + 1]], want, torch.float32, limit=1e-6)
        assert state[slot].item() == mine[-1]
    alone = kernels.embed_pairs(table.to(dtype).to(CUDA), ints(tokens), positions=ints(positions), **entries)
    close(alone, table[tokens], torch.float32, limit=1e-7)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8, 11])
@pytest.mark.parametrize("width", [50, 64, 384, 4096])
def test_streams_are_written_read_and_normed_in_one_pass(width, streams, dtype):
    """The write behind a sublayer (one output, or a pair still to be normed and added up, with and without biases)
    and the norm in front of the next, from streams that differ and from streams that are still one; on gathered
    rows nothing is written and the sum of the streams is normed."""
    from tinyvllm_b200.ops import kernels
    from tinyvllm_b200.parts.hyper import NormedPair

    g = torch.Generator().manual_seed(width + streams)
    tokens, eps = 7, 1e-5
    f32 = lambda *shape, spread=1.0: (torch.randn(*shape, generator=g) * spread).float()
    dev = lambda t: t.float().contiguous().to(CUDA)
    w_in, w_mix, w_out = f32(streams), f32(streams, streams), f32(streams)
    weight, bias = 1.0 + f32(width, spread=0.3), f32(width, spread=0.3)
    left, right = rounded(f32(tokens, width, spread=5.0), dtype), rounded(f32(tokens, width, spread=0.2), dtype)
    wl, wr, bl, br = 1.0 + f32(width, spread=0.3), 1.0 + f32(width, spread=0.3), f32(width), f32(width, spread=0.1)
    y = f32(tokens, width, spread=4.0)
    limit = 1.2e-5 if dtype == torch.float32 else 6e-3       # sums over 4,096 terms in another order
    for spread in (False, True):
        x = f32(tokens, width, spread=3.0) if spread else f32(tokens, streams, width, spread=3.0)
        full = x.double()[:, None, :].repeat(1, streams, 1) if spread else x.double()
        # read alone
        out, same = kernels.hyper_norm(dev(x), streams=streams, w_in=dev(w_in), weight=dev(weight), bias=dev(bias),
                                       eps=eps, out_dtype=dtype)
        want = plain.layer_norm(plain.read_streams(full, w_in.double()), weight.double(), bias.double(), eps)
        close(out, want, dtype, limit=limit)
        close(same, x, torch.float32, limit=1e-9)
        for kind in ("one", "pair", "pair with biases"):
            if kind == "one":
                update, added = dev(y), y.double()
            else:
                biases = kind != "pair"
                update = NormedPair(left.to(dtype).to(CUDA), right.to(dtype).to(CUDA), left_weight=dev(wl),
                                    right_weight=dev(wr), left_bias=dev(bl) if biases else None,
                                    right_bias=dev(br) if biases else None, eps=eps, factor=0.5)
                added = plain.half_sum_of_normed(left + (bl.double() if biases else 0.0),
                                                 right + (br.double() if biases else 0.0), wl.double(), wr.double(), eps)
                close(update.materialise(), added, torch.float32, limit=2e-6)
            new = plain.write_streams(full, added, w_mix.double(), w_out.double())
            stream = dev(x)
            out, updated = kernels.hyper_norm(stream, streams=streams, w_in=dev(w_in), weight=dev(weight), bias=dev(bias),
                                              eps=eps, out_dtype=dtype, y=update, w_mix=dev(w_mix), w_out=dev(w_out))
            assert (updated is stream) == (not spread)
            close(updated, new, torch.float32, limit=2e-6)
            want = plain.layer_norm(plain.read_streams(new, w_in.double()), weight.double(), bias.double(), eps)
            close(out, want, dtype, limit=limit)
            again = dev(x)
            some, nothing = kernels.hyper_norm(again, streams=streams, w_in=None, weight=dev(weight), bias=dev(bias),
                                               eps=eps, out_dtype=dtype, y=update, w_mix=dev(w_mix), w_out=dev(w_out),
                                               rows=ints([5, 0, 5]))
            assert nothing is None and torch.equal(again.cpu(), x)
            close(some, plain.layer_norm(new.sum(1), weight.double(), bias.double(), eps)[[5, 0, 5]], dtype, limit=limit)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("taps,channels", [(1, 12), (2, 64), (3, 37), (4, 256), (5, 130), (8, 40), (9, 72), (16, 20), (31, 8)])
def test_short_convolution_from_carried_inputs(taps, channels, dtype):
    """A long portion, portions shorter than the taps, single tokens and a padding row, from the inputs earlier tokens
    left; one input of a hundred far inside is seen by exactly the next ``taps`` outputs."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(taps * 100 + channels)
    kernel_taps = next(k for k in kernels.CONV_TAPS if k >= taps)
    lengths, slots = [101, 2, 1, 40, 3, 1, 1], [2, 6, 0, 5, 1, 3, 4]
    entries, starts = entries_of(lengths, slots, padding=(5,))
    at = 4 if channels % 4 == 0 else 3
    proj = rounded(torch.randn(starts[-1], channels + 8, generator=g), dtype)
    proj[60, at:at + channels] = 100.0
    w, bias = torch.randn(channels, taps, generator=g).float(), torch.randn(channels, generator=g).float()
    by_tap = torch.zeros(kernel_taps, channels)
    by_tap[kernel_taps - taps:] = w.t()
    state = rounded(torch.randn(7, kernel_taps - 1, channels, generator=g), dtype).float()
    device_state = state.to(CUDA)
    x = proj.to(dtype).to(CUDA)[:, at:at + channels]
    got = kernels.short_convolution(x, by_tap.to(CUDA), bias=bias.to(CUDA), act="silu", state=device_state, **entries)
    want_state = state.double().clone()
    for r, slot in enumerate(slots):
        rows = slice(starts[r], starts[r + 1])
        if r == 5:
            assert (got[rows] == 0).all()
            continue
        y, tail = plain.causal_convolution(proj[rows, at:at + channels], by_tap.t().double(), bias.double(),
                                           state[slot].double())
        close(got[rows], plain.silu(y), dtype, scale=max(1.0, y.abs().max().item()), limit=4e-6 if dtype == torch.float32 else 6e-3)
        want_state[slot] = tail
    close(device_state, want_state, torch.float32, limit=1e-9)
    plainly, _ = plain.causal_convolution(proj[:101, at:at + channels], by_tap.t().double(), bias.double(), state[2].double())
    proj[60, at:at + channels] = 0.0
    without, _ = plain.causal_convolution(proj[:101, at:at + channels], by_tap.t().double(), bias.double(), state[2].double())
    moved = ((plainly - without).abs().amax(1) > 1e-9).nonzero().flatten().tolist()
    assert moved == list(range(60, min(60 + taps, 101)))


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("channels,n,rank", [(64, 16, 8), (37, 7, 5), (130, 33, 20), (64, 1, 1), (40, 3, 2), (31, 20, 3), (512, 16, 16),
                                             (72, 40, 9), (48, 24, 12), (20, 64, 8), (40, 128, 4), (24, 100, 6), (16, 256, 2)])
def test_selective_scan_from_a_carried_state(channels, n, rank, dtype):
    """Five entries of one step from carried states, with every number of lanes; then three steps of single tokens in
    the one-launch form, with the step sizes' product done inside and outside, beside the scan.  Channel 0 takes
    token 2 in (a large step size there, almost none elsewhere) and must still hold it 400 tokens later."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(channels * 10 + n)
    lengths, slots = [403, 40, 1, 1, 2], [3, 0, 5, 1, 4]
    entries, starts = entries_of(lengths, slots)
    tokens = starts[-1]
    f32 = lambda *shape, spread=1.0: (torch.randn(*shape, generator=g) * spread).float()
    a = -torch.exp(torch.rand(channels, n, generator=g) * 4.0 - 3.0).float()
    a[0] = -0.01
    d, dt_bias = f32(channels), torch.rand(channels, generator=g) * 5.0 - 5.0
    x, z = rounded(f32(tokens, channels + 2), dtype), rounded(f32(tokens, channels + 4), dtype)
    bc = rounded(f32(tokens, 2 * n + 3), dtype)
    pre = f32(tokens, channels)
    pre[:, 0], pre[2, 0], dt_bias[0] = -30.0, 8.0, 0.0
    bc[402, n:2 * n] = bc[2, :n]                                   # the query of token 402 is token 2's direction
    xs, zs, b, c = x[:, 1:1 + channels], z[:, 3:3 + channels], bc[:, :n], bc[:, n:2 * n]
    dt = plain.softplus(pre.double() + dt_bias.double())
    state = f32(6, channels, n, spread=0.3)
    state[3] = 0.0
    want, want_state, far = torch.zeros(tokens, channels, dtype=F64), state.double().clone(), None
    for r, slot in enumerate(slots):
        rows = slice(starts[r], starts[r + 1])
        y, want_state[slot] = plain.selective_scan(xs[rows], dt[rows], b[rows], c[rows], a.double(), d.double(), state[slot].double())
        want[rows] = y * plain.silu(zs[rows])
        if r == 0:
            far = (dt[2, 0] * xs[2, 0] * torch.exp(-0.01 * dt[3:403, 0].sum()) * (b[2] * b[2]).sum(), y[402, 0] - d[0].double() * xs[402, 0])
    assert abs(far[0] - far[1]) < 0.02 * abs(far[0])               # what channel 0 reads at token 402 is token 2
    dev = lambda t, kind=torch.float32: t.to(kind).to(CUDA)
    dx, dz, dbc = dev(x, dtype), dev(z, dtype), dev(bc, dtype)
    common = dict(a=dev(a), d=dev(d), dt_bias=dev(dt_bias))
    limit = 2e-5 if dtype == torch.float32 else None
    fewest = 2 if n <= 2 else 4 if n <= 4 else 8 if n <= 128 else 16
    for lanes, tile in [(0, 0)] + [(lanes, tile) for lanes in sorted({fewest, 16 if n > 8 else fewest}) for tile in (1, 2)
                                   if tile == 1 or (lanes >= 8 and lanes * 8 >= n)]:
        device_state = dev(state)
        out = torch.full((tokens, channels + 5), 7.0, dtype=dtype, device=CUDA)
        kernels.selective_scan(dx[:, 1:1 + channels], pre=dev(pre), z=dz[:, 3:3 + channels], b=dbc[:, :n], c=dbc[:, n:2 * n],
                               state=device_state, out=out[:, 2:2 + channels], lanes=lanes, tile=tile, **common, **entries)
        close(out[:, 2:2 + channels], want, dtype, limit=limit)
        close(device_state, want_state, torch.float32, limit=3e-5)
        assert torch.equal(device_state[2].cpu(), state[2]) and (out[:, :2] == 7.0).all() and (out[:, 2 + channels:] == 7.0).all()
    # single tokens: seven rows, one of them padding
    wide = -(-rank // 8) * 8
    w = torch.zeros(channels, wide, dtype=F64)
    w[:, :rank] = rounded(f32(channels, rank, spread=0.5), dtype)
    slots = [5, 2, 7, 0, 6, 1, 3]
    for rows_count, padding in ((7, (3,)), (21, (20,))):
        all_slots = slots if rows_count == 7 else list(range(21))
        entries, _ = entries_of([1] * rows_count, all_slots, padding)
        state = f32(21 if rows_count == 21 else 8, channels, n, spread=0.5)
        inside, outside, scanned = dev(state), dev(state), dev(state)
        want_state = state.double().clone()
        for _ in range(3):
            row = wide + 2 * n
            mixed = rounded(f32(rows_count, row + 3), dtype)
            xs, zs = rounded(f32(rows_count, channels), dtype), rounded(f32(rows_count, channels), dtype)
            pre = mixed[:, :wide] @ w.T
            dt = plain.softplus(pre + dt_bias.double())
            want = torch.zeros(rows_count, channels, dtype=F64)
            for r in range(rows_count):
                if r in padding:
                    continue
                slot = all_slots[r]
                y, want_state[slot] = plain.selective_scan(xs[r:r + 1], dt[r:r + 1], mixed[r:r + 1, wide:wide + n],
                                                           mixed[r:r + 1, wide + n:row], a.double(), d.double(), want_state[slot])
                want[r] = (y * plain.silu(zs[r:r + 1]))[0]
            dm = dev(mixed, dtype)
            given = dict(z=dev(zs, dtype), b=dm[:, wide:wide + n], c=dm[:, wide + n:row], **common, **entries)
            for device_state, more in ((inside, dict(pre=None, low=dm[:, :wide], dt_weight=dev(w, dtype), single=True)),
                                       (outside, dict(pre=dev(pre), single=True)), (scanned, dict(pre=dev(pre)))):
                out = torch.full((rows_count, channels), 7.0, dtype=dtype, device=CUDA)
                kernels.selective_scan(dev(xs, dtype), out=out, state=device_state, **more, **given)
                close(out, want, dtype, limit=limit)
                close(device_state, want_state, torch.float32, limit=3e-5)
                assert (out[list(padding)] == 0).all()
        free = [s for s in range(state.shape[0]) if s not in all_slots] + [all_slots[p] for p in padding]
        assert torch.equal(inside[free].cpu(), state[free])


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,dim,vdim,tau,rank", [(4, 16, 32, 12.0, 16), (3, 10, 7, 5.0, 5), (2, 6, 20, 1.0, 3),
                                                     (2, 130, 48, 16.0, 8), (1, 5, 3, 3.0, 1), (2, 64, 128, 16.0, 16), (1, 256, 40, 2.0, 24)])
def test_decayed_linear_attention_from_a_carried_state(heads, dim, vdim, tau, rank, dtype):
    """Five entries from carried states, as whole entries and in pieces of several sizes, then single tokens in the
    one-launch form with the decays' second step done inside.  Channel 0 of head 0 keeps everything and is written by
    token 2 alone; the query 400 tokens later reads along it and must find token 2's value."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(heads * 1000 + dim)
    per, hv, wide = heads * dim, heads * vdim, -(-rank // 8) * 8
    q_at, k_at, v_at, g_at, low_at = 1, 2 + per, 3 + 2 * per, 4 + 2 * per + hv, 5 + 2 * per + 2 * hv
    cols = low_at + wide
    lengths, slots = [403, 40, 1, 1, 2], [3, 0, 5, 1, 4]
    entries, starts = entries_of(lengths, slots)
    tokens = starts[-1]
    a2 = torch.zeros(per, wide, dtype=F64)
    a2[:, :rank] = rounded(torch.randn(per, rank, generator=g), dtype)
    a2[0] = 0.0
    bias = (torch.rand(per, generator=g) * 8.0 - 1.0).float()
    bias[0] = 60.0
    weight = (1.0 + 0.2 * torch.randn(vdim, generator=g)).float()
    scale, eps = dim ** -0.5, 1e-5

    def project(count):
        return rounded(torch.randn(count, cols, generator=g), dtype)

    def reference(proj, state):
        q, k = (proj[:, at:at + per].view(-1, heads, dim) for at in (q_at, k_at))
        v = proj[:, v_at:v_at + hv].view(-1, heads, vdim)
        z = proj[:, low_at:] @ a2.T + bias.double()
        o, state = plain.decayed_linear_attention(q * scale, k, v, (torch.sigmoid(z) ** (1.0 / tau)).view(-1, heads, dim), state)
        out = plain.rms_norm(o, weight.double(), eps).reshape(-1, hv) * plain.silu(proj[:, g_at:g_at + hv])
        return out, o, state, z - bias.double()

    proj = project(tokens)
    proj[:403, k_at] = 0.0
    proj[2, k_at] = 6.0
    proj[402, q_at:q_at + dim] = 0.0
    proj[402, q_at] = 5.0
    state = (torch.randn(6, heads, dim, vdim, generator=g) * 0.3).float()
    state[3] = 0.0
    want, want_state, gates = [], state.double().clone(), []
    for r, slot in enumerate(slots):
        out, o, want_state[slot], z = reference(proj[starts[r]:starts[r + 1]], state[slot].double())
        want.append(out)
        gates.append(z)
        if r == 0:
            v2 = proj[2, v_at:v_at + vdim]
            assert (o[402, 0] @ v2) / (o[402, 0].norm() * v2.norm()) > 0.99
    want = torch.cat(want)
    common = dict(q_at=q_at, g_at=-1, k_at=k_at, v_at=v_at, heads=heads, dim=dim, vdim=vdim, bias=bias.to(CUDA),
                  query_act=None, query_scale=scale, gate_exponent=1.0 / tau, unit_norm=True,
                  norm_weight=weight.to(CUDA), eps=eps, out_gate_at=g_at)
    gate_pre = torch.cat(gates).float().to(CUDA)
    # a norm over a head multiplies what cancelled in the head's sum: the bound is on the scale of all heads
    limit = 5e-5 if dtype == torch.float32 else None
    for segment in (0, 5, 64, 403, None):
        device_state = state.to(CUDA)
        got = kernels.gated_recurrence(proj.to(dtype).to(CUDA), state=device_state, gate_pre=gate_pre, segment=segment,
                                       **common, **entries)
        close(got, want, dtype, limit=limit)
        close(device_state, want_state, torch.float32, limit=3e-5)
        assert torch.equal(device_state[2].cpu(), state[2])
    slots = [5, 2, 7, 0, 6, 1, 3]
    entries, _ = entries_of([1] * 7, slots, padding=(3,))
    state = (torch.randn(8, heads, dim, vdim, generator=g) * 0.5).float()
    inside, outside = state.to(CUDA), state.to(CUDA)
    want_state = state.double().clone()
    for _ in range(3):
        proj = project(7)
        want = torch.zeros(7, hv, dtype=F64)
        pre = torch.zeros(7, per, dtype=F64)
        for r in range(7):
            if r != 3:
                want[r:r + 1], _, want_state[slots[r]], pre[r:r + 1] = reference(proj[r:r + 1], want_state[slots[r]])
        device = proj.to(dtype).to(CUDA)
        for device_state, more in ((inside, dict(low_at=low_at, low_weight=a2.to(dtype).to(CUDA))),
                                   (outside, dict(gate_pre=pre.float().to(CUDA)))):
            got = kernels.gated_recurrence(device, state=device_state, **more, **common, **entries)
            close(got, want, dtype, limit=limit)
            close(device_state, want_state, torch.float32, limit=3e-5)
            assert (got[3] == 0).all()
    assert torch.equal(inside[[4, 0]].cpu(), state[[4, 0]])


def paged(keys, values, page, dtype, seed, fill):
    """Keys [n, kv, dk] and values [n, kv, dv] of one request spread over shuffled pages."""
    n, kv, dk = keys.shape
    count = -(-n // page)
    order = list(range(count + 3))
    random.Random(seed).shuffle(order)
    table = order[:count]
    key_cache = torch.full((count + 3, kv, page, dk), fill, dtype=dtype)
    value_cache = torch.full((count + 3, kv, page, values.shape[2]), fill, dtype=dtype)
    for j in range(n):
        key_cache[table[j // page], :, j % page] = keys[j].to(dtype)
        value_cache[table[j // page], :, j % page] = values[j].to(dtype)
    return key_cache.to(CUDA), value_cache.to(CUDA), torch.tensor([table], dtype=torch.int32, device=CUDA)


# (query position, key that is made to stand out for it): far back, at both sides of page borders and of the borders
# between chunks of 32, 128 and 256 keys that the kernels cut the keys in, the query itself, the first token
STANDOUTS = {700: 3, 699: 255, 698: 256, 697: 248, 696: 247, 695: 695, 0: 0, 1: 0, 300: 299, 130: 127, 129: 128, 97: 96, 94: 31}


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("kind", ["rows", "split", "tiles", "singles"])
@pytest.mark.parametrize("softcap", [14.0, 40.0, 3000.0])
@pytest.mark.parametrize("heads,kv,dk,dv", [(4, 2, 16, 32), (3, 1, 12, 5), (8, 8, 32, 16), (40, 2, 16, 16), (9, 3, 48, 80),
                                            (4, 2, 64, 128), (2, 1, 128, 64)])
def test_attention_with_capped_scores(heads, kv, dk, dv, softcap, kind, dtype):
    """Random scores of a few units plus one key per checked query whose score is a hundred: a cap of 14 brings it down to
    the cap, where it shares the weight with the others by e^14 (and one half of the queries see twelve such keys
    share alike); a wide cap leaves it all the weight.  Ordinary scores are bent as the cap says."""
    from tinyvllm_b200.ops import kernels

    if kind in ("tiles", "singles") and (dtype != torch.bfloat16 or dk % 16 or dv % 16):
        pytest.skip("the tensor-core kernels take bfloat16 and sizes in steps of 16")
    n, page, scale = 701, 8, 0.4
    g = torch.Generator().manual_seed(heads * 100 + dk)
    q = torch.randn(n, heads, dk, generator=g) * (8.0 / dk ** 0.5)
    k = torch.randn(n, kv, dk, generator=g)
    v = torch.randn(n, kv, dv, generator=g)
    axis = {key: i for i, key in enumerate(sorted(set(STANDOUTS.values())))}
    for key, i in axis.items():
        k[key, 0] = 0.0
        k[key, 0, i % dk] = 62.5
    for query, key in STANDOUTS.items():
        if query != key:
            q[query, 0] = 0.0
            q[query, 0, axis[key] % dk] = 4.0
    q, k, v = rounded(q, dtype), rounded(k, dtype), rounded(v, dtype)
    rows = sorted(STANDOUTS)
    shared = [h // (heads // kv) for h in range(heads)]
    s = plain.capped_scores(q[rows], k[:, shared], scale, softcap)
    visible = torch.arange(n)[None, :] <= torch.tensor(rows)[:, None]
    weights = torch.softmax(s.masked_fill(~visible[None], -torch.inf), -1)
    want = torch.einsum("hij,jhv->ihv", weights, v[:, shared])
    uncapped = torch.softmax(plain.capped_scores(q[rows], k[:, shared], scale, None).masked_fill(~visible[None], -torch.inf), -1)
    bent = (torch.einsum("hij,jhv->ihv", uncapped, v[:, shared]) - want).abs().max().item()
    assert bent > 0.05 or softcap > 1000                           # forgetting the cap would show
    key_cache, value_cache, block_table = paged(k, v, page, dtype, 3, float("nan") if kind in ("rows", "split") else 1e30)
    flat = lambda t, sel: t[sel].to(dtype).reshape(len(sel), -1).to(CUDA)
    everything = list(range(n))
    if kind in ("rows", "split"):
        chunks = 3 if kind == "split" else 0
        scratch = torch.empty(kernels.attention_rows_scratch_floats(len(rows), heads, dv, 3), dtype=torch.float32,
                              device=CUDA) if chunks else None
        got = kernels.attention_rows(
            flat(q, rows), heads * dk, key_cache, value_cache, block_table, ints([0] * len(rows)), ints(rows),
            num_q=heads, num_kv=kv, head_dim=dk, value_dim=dv, window=None, scale=scale, scratch=scratch,
            max_chunks=chunks, softcap=softcap)
    elif kind == "tiles":
        firsts = [0, 1, 3, 50] + list(range(114, n, 64))          # tiles of up to 64 tokens, cut at odd places
        counts = [b - a for a, b in zip(firsts, firsts[1:] + [n])]
        out = torch.empty(n, heads * dv, dtype=dtype, device=CUDA)
        kernels.attention_tiles(
            flat(q, everything), key_cache, value_cache, block_table, ints(everything), ints([0] * len(firsts)),
            ints(firsts), ints(counts), num_q=heads, num_kv=kv, key_dim=dk, value_dim=dv, window=None, keep_first=0,
            scale=scale, out=out, softcap=softcap)
        got = out[rows]
    else:
        got = torch.empty(len(rows), heads * dv, dtype=dtype, device=CUDA)
        need = kernels.attention_tiles_singles_floats(len(rows), heads, dv, None, 0, 704)
        kernels.attention_tiles_singles(
            flat(q, rows), key_cache, value_cache, block_table, ints(rows), ints([0] * len(rows)), num_q=heads,
            num_kv=kv, key_dim=dk, value_dim=dv, window=None, keep_first=0, scale=scale, max_context=704,
            scratch=torch.empty(need, dtype=torch.float32, device=CUDA), out=got, softcap=softcap)
    close(got.view(len(rows), heads, dv), want, dtype, scale=want.abs().max().item(),
          limit=3e-5 if dtype == torch.float32 else None)


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("heads,kv,dim,vdim,rot", [(4, 2, 16, 32, 8), (3, 1, 9, 5, 4), (8, 8, 32, 16, 32), (1, 1, 7, 7, 2),
                                                   (8, 2, 64, 64, 32), (8, 2, 128, 128, 128), (4, 4, 64, 128, 48), (2, 2, 256, 24, 64),
                                                   (2, 1, 24, 40, 0)])
@pytest.mark.parametrize("tokens", [9, 130])
def test_biases_and_paired_halves_go_to_the_cache(tokens, heads, kv, dim, vdim, rot, dtype):
    """q, k and v get their biases, q and k turn as paired halves by their positions, q in place, k and v in the
    token's cache rows; a token without a slot (a padding row) stores nothing.  Few and many tokens take different
    kernels where the sizes allow the wide one."""
    from tinyvllm_b200.ops import kernels

    g = torch.Generator().manual_seed(heads * 10 + dim)
    page = 4
    positions = torch.tensor([0, 1, 2, 3, 250, 251, 40, 7, 1000] + list(range(300, 300 + tokens - 9)))
    slots = [5, 6, 7, 8, 0, 1, -1, 14, 19] + list(range(20, 20 + tokens - 9))
    pages = -(-(tokens + 11) // page)
    q_cols, k_cols, v_cols = heads * dim, kv * dim, kv * vdim
    at = 8 if dim % 8 == 0 else 3
    proj = rounded(torch.randn(tokens, at + q_cols + k_cols + v_cols, generator=g) * 2.0, dtype)
    qb, kb, vb = (torch.randn(c, generator=g).float() for c in (q_cols, k_cols, v_cols))
    q = (proj[:, at:at + q_cols] + qb.double()).view(tokens, heads, dim)
    k = (proj[:, at + q_cols:at + q_cols + k_cols] + kb.double()).view(tokens, kv, dim)
    v = (proj[:, at + q_cols + k_cols:] + vb.double()).view(tokens, kv, vdim)
    inv_freq = None
    if rot:
        rotation = {"dims": rot, "base": 77.0}
        q, k = plain.rotate_halves(q, positions, rotation), plain.rotate_halves(k, positions, rotation)
        inv_freq = torch.tensor([77.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=F64).float().to(CUDA)
    device = proj.to(dtype).to(CUDA)
    keys = torch.full((pages, kv, page, dim), 9.0, dtype=dtype, device=CUDA)
    values = torch.full((pages, kv, page, vdim), 9.0, dtype=dtype, device=CUDA)
    kernels.qkv_prepare(device, q_at=at, k_at=at + q_cols, v_at=at + q_cols + k_cols, num_q=heads, num_kv=kv, key_dim=dim,
                        value_dim=vdim, positions=ints(positions.tolist()), inv_freq=inv_freq, rot_dims=rot,
                        pairing="half_split", slots=ints(slots), key_cache=keys, value_cache=values, q_bias=qb.to(CUDA),
                        k_bias=kb.to(CUDA), v_bias=vb.to(CUDA))
    limit = 2e-4 if dtype == torch.float32 else 8e-3             # float32 angles at position 1,000
    close(device[:, at:at + q_cols], q.reshape(tokens, -1), dtype, limit=limit)
    assert torch.equal(device[:, :at].cpu().double(), proj[:, :at])
    written = torch.zeros(pages * page, dtype=torch.bool)
    for t, slot in enumerate(slots):
        if slot >= 0:
            written[slot] = True
            close(keys[slot // page, :, slot % page], k[t], dtype, limit=limit)
            close(values[slot // page, :, slot % page], v[t], dtype, limit=limit)
    assert (keys.permute(0, 2, 1, 3).reshape(pages * page, -1)[~written] == 9.0).all()
    assert (values.permute(0, 2, 1, 3).reshape(pages * page, -1)[~written] == 9.0).all()


# ------------------------------------------------------- parts outside the blocks this design puts them in
@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_the_mixers_stand_alone_too(dtype):
    """The scan and the attention with an output bias as mixers of their own (their own input and output products),
    and the pair of mixers added up by its own kernel, over a step of two entries."""
    from tinyvllm_b200.cache.storage import CacheStorage, group_runs
    from tinyvllm_b200.config.spec import PartSpec
    from tinyvllm_b200.parts import BuildContext, build_part
    from tinyvllm_b200.weights.loader import bind_tensors
    from zifunex_configs import tensors_of

    name = "e"
    config = ZIFUNEX_CONFIGS[name]
    tensors = {k: v.to(torch.bfloat16) for k, v in tensors_of(config, 3).items()}
    w = {k: v.double() for k, v in tensors.items()}
    pair = config.to_spec().layers[0].mixer
    specs = {"left": pair.params["left"], "right": pair.params["right"], "": pair}
    g = torch.Generator().manual_seed(5)
    lengths = [50, 17]
    x = rounded(torch.randn(sum(lengths), config.width, generator=g), dtype)
    for which, spec in specs.items():
        at = "l0.mix" + (f".{which}" if which else "")
        part = build_part("mixer", PartSpec(spec.kind, {**spec.params}), BuildContext(torch.device(CUDA), dtype, at))
        targets = [(p, s) for p in part.all_parts() for s in p.param_specs()]
        names = {source.name for _, s in targets for source in s.sources}
        bind_tensors(targets, {k: v for k, v in tensors.items() if k in names}, dtype=dtype, device=CUDA)
        for p in part.all_parts():
            if hasattr(p, "finalize"):
                p.finalize()
        needs = [part.cache_need()]
        groups, where = group_runs(needs, [None])
        storage = CacheStorage(groups, where, needs, page_size=8, pages_per_group=12, num_state_slots=3, dtype=dtype, device=CUDA)
        entries, starts = entries_of(lengths, [2, 0])
        positions = [i for n in lengths for i in range(n)]
        slots = [i for i in range(50)] + [56 + i for i in range(17)]
        table = torch.full((2, 8), -1, dtype=torch.int32)
        table[0, :7], table[1, :3] = torch.arange(7), torch.arange(7, 10)
        ctx = SimpleNamespace(storage=storage, num_tokens=67, num_rows=2, positions=ints(positions), slots=[ints(slots)],
                              block_tables=[table.to(CUDA)], max_position=49, max_context=96, split_chunks=0,
                              decode_only=False, tile_row=None, single_runs=(), writes_cache=lambda run: True, shared={}, **entries)
        got = part.forward(x.to(dtype).to(CUDA), ctx, 0)
        mixer = config.to_json()["layers"][0]["mixer"]
        for r in range(2):
            rows = slice(starts[r], starts[r + 1])
            if which == "left":
                want = plain.softcapped_attention(x[rows], w, at, mixer["left"])
            elif which == "right":
                want = plain.mamba(x[rows], w, at, mixer["right"])[0]
            else:
                want = plain.parallel(x[rows], w, at, mixer, config.norm_eps)
            close(got[rows], want, dtype, limit=2e-5 if dtype == torch.float32 else 2.5e-2)


# ---------------------------------------------------------------- whole models
def requests_of(name):
    vocab = ZIFUNEX_CONFIGS[name].vocab
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
    the rounding of 16-bit activations.  The others are tokens whose linear attention nearly cancels: the norm over a
    head gives o = S^T q the same size however small it is, so where q is nearly orthogonal to what the state holds
    (at a request's first token, to its own key) rounding decides the direction of a whole head (observed: 0.7 of the
    scale at a first token whose q . k is 0.0005 of the sum of its terms' sizes)."""
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
        assert median <= 1.5e-2 and most <= 5e-2, \
            f"median {median:.3g}, ninth decile {most:.3g} of the largest logit, worst at {worst[1:]}"


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
@pytest.mark.parametrize("name", sorted(ZIFUNEX_CONFIGS))
@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed"])
def test_every_way_of_cutting_gives_the_plain_logits(cut, name, dtype, folders):
    """Whole prompts; prompts whose last 40 tokens come one by one; portions of changing size down to two tokens, cut
    inside pages, convolutions and blocks of the scans; up to four live requests with portions beside single tokens,
    in a pool with room for little more than the live tokens and four state slots, so that pages and slots that
    finished requests gave back are taken again."""
    requests = requests_of(name)
    page = ZIFUNEX_PAGES[name]
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


@pytest.mark.parametrize("dtype", DTYPES, ids=IDS)
def test_a_request_is_not_moved_by_its_neighbours(dtype, folders):
    """The same request alone and beside three others, in other pages and another state slot: equal beyond
    rounding."""
    name = "a"
    requests = requests_of(name)
    page = ZIFUNEX_PAGES[name]
    alone = {"x": requests["a150"]}
    with torch.inference_mode():
        first = rh.run_steps(make_runner(folders[name], dtype, page, 64), rh.portions(alone, 9, sizes=(7, 50)))
        crowd = dict(list(requests.items())[2:])
        crowd["x"] = requests["a150"]
        second = rh.run_steps(make_runner(folders[name], dtype, page, 96), rh.mixed(crowd, 1, live=4, decode_tail=5))
    scale = oracle_logits(folders[name], alone)["x"].abs().max().item()
    worst = max((first[key].double() - second[key].double()).abs().max().item() / scale for key in first)
    assert worst <= (2e-5 if dtype == torch.float32 else 4e-2)


def test_a_slot_that_is_taken_again_starts_from_zero(folders):
    """One state slot and pages for one request: the second request gets the slot and the pages the first
    one left, and its logits are those of a request that runs alone in a fresh pool (a pair row, a convolution or a
    state of the request before would show at its first tokens)."""
    name = "d"
    vocab = ZIFUNEX_CONFIGS[name].vocab
    requests = {"one": tokens_of(vocab, 50, 1), "two": tokens_of(vocab, 45, 2)}
    runner = make_runner(folders[name], torch.float32, 4, 13, max_len=52, max_requests=1)
    with torch.inference_mode():
        got = rh.run_steps(runner, rh.portions(requests, 6, sizes=(2, 11, 30)))
    compare(got, folders[name], requests, torch.float32)


@pytest.mark.parametrize("name", ["a", "b", "f"])
def test_long_decoding(name, folders):
    """A prompt of five tokens and 330 tokens decoded one by one, float32: states, convolutions and pairs run along
    335 tokens."""
    tokens = tokens_of(ZIFUNEX_CONFIGS[name].vocab, 335, 9)
    requests = {"long": tokens}
    page = ZIFUNEX_PAGES[name]
    runner = make_runner(folders[name], torch.float32, page, 352 // page, max_len=352)
    with torch.inference_mode():
        got = rh.run_steps(runner, rh.tail_by_one(requests, 330))
    compare(got, folders[name], requests, torch.float32)


@pytest.mark.parametrize("dtype_name", ["float32", "bfloat16"])
def test_trace_program(dtype_name, folders, tmp_path):
    name = "b"
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
    got = rh.read_trace_output(steps, out, ZIFUNEX_CONFIGS[name].vocab)
    compare(got, folders[name], requests, getattr(torch, dtype_name))


@pytest.mark.parametrize("eager", [True, False], ids=["eager", "graphs"])
@pytest.mark.parametrize("name", sorted(ZIFUNEX_CONFIGS))
def test_greedy_generation_through_the_engine(name, eager, folders):
    """LLM.generate (scheduler, chunked prefill, decode graphs and runs of decode steps) against greedy
    decoding with the plain implementation, float32."""
    from tinyvllm_b200 import LLM, EngineConfig, SamplingParams

    config = ZIFUNEX_CONFIGS[name]
    prompts = [tokens_of(config.vocab, n, 700 + n) for n in (1, 9, 40, 77, 130)]
    engine_config = EngineConfig(
        model=folders[name], dtype="float32", max_model_len=512, max_num_seqs=4, max_num_batched_tokens=64,
        prefill_chunk_size=24, kv_block_size=ZIFUNEX_PAGES[name], kv_cache_memory_bytes=16 * 1024 * 1024,
        prefill_reserve_tokens=0, prefill_reserve_requests=0, enforce_eager=eager)
    with LLM(engine_config) as llm:
        outputs = llm.generate(prompts, SamplingParams(max_new_tokens=20, ignore_eos=True))
        if not eager:
            assert llm.engine.graph_steps > 0
    for prompt, output in zip(prompts, outputs):
        assert list(output.output_token_ids) == greedy_oracle(folders[name], prompt, 20)


def test_steps_whose_shape_comes_back_replay_from_the_right_state(folders):
    """Prompts cut into equal portions: from their third occurrence on the steps are captured and replayed; a step that
    is run a second time to be captured starts from the states (the token before among them) it started from."""
    from tinyvllm_b200 import LLM, EngineConfig, SamplingParams

    name = "a"
    config = ZIFUNEX_CONFIGS[name]
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

    name = "a"
    config = ZIFUNEX_CONFIGS[name]
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
        if (top[0] - top[1]).item() > 0.05 * logits.abs().max().item():
            assert output.output_token_ids[0] == int(logits.argmax())


def test_bfloat16_steps_run_on_the_tensor_core_and_one_launch_kernels(folders, monkeypatch):
    """Head sizes in steps of 16: prompt portions go to the tile kernel, decoded tokens to the kernel for single tokens,
    none to the row kernel, all with the cap; decoded tokens move both recurrences' states in one launch."""
    from tinyvllm_b200.ops import kernels

    seen = {"attention_tiles": [], "attention_tiles_singles": [], "attention_rows": [], "selective_scan": [],
            "gated_recurrence": []}
    for fn in seen:
        original = getattr(kernels, fn)

        def watched(*args, _original=original, _fn=fn, **kwargs):
            seen[_fn].append(kwargs.get("softcap") if "attention" in _fn else
                             bool(kwargs.get("single")) if _fn == "selective_scan" else kwargs.get("low_at") is not None)
            return _original(*args, **kwargs)
        monkeypatch.setattr(kernels, fn, watched)
    name = "e"
    config = ZIFUNEX_CONFIGS[name]
    requests = {"t": tokens_of(config.vocab, 90, 31)}
    runner = make_runner(folders[name], torch.bfloat16, 16, 16)
    with torch.inference_mode():
        rh.run_steps(runner, rh.tail_by_one(requests, 3))
    runs = [config.layers[i] for i in config.run_order()]
    caps = [layer.left.softcap for layer in runs if layer.left is not None]
    linear = len(runs) - len(caps)
    assert seen["attention_tiles"] == caps                       # one prompt step
    assert seen["attention_tiles_singles"] == caps * 3           # three decoded tokens
    assert not seen["attention_rows"]
    assert seen["selective_scan"] == [False] * len(caps) + [True] * len(caps) * 3
    assert seen["gated_recurrence"] == [False] * linear + [True] * linear * 3


def test_command_line(folders, capsys):
    """python -m tinyvllm_b200 on a Zifunex folder: greedy tokens of the plain implementation, also
    streamed, and with weights drawn from a seed instead of the file."""
    from tinyvllm_b200.__main__ import main

    name = "b"
    prompts = [tokens_of(ZIFUNEX_CONFIGS[name].vocab, n, 950 + n) for n in (3, 45)]
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

"""Small Zifunex configurations for the tests, their weights and their oracle.

The configurations differ in everything config.json can say: width, vocabulary, 1 to 6 streams, number and order of
layers (each mixer comes first somewhere), loops over the middle, the start and the end, once and several times, and
none; attention with 1, 2, 3 and 4 query heads a kv head, key and value sizes that are equal or not, multiples of 16
or odd, rotation over a part of a head, over all of it or none, tight, loose and no caps on the scores; scans with
states of 1 to 40 numbers, fewer and more channels than the width, low-rank parts of 1 to 20, convolutions of 1 to 9
taps; linear attention with key sizes from 5 to 130, decays whose root is taken or not (an exponent of 1), decay
projections of rank 3 to 16; layers with and without a feed-forward; pair tables of a few and of many rows; models
of linear attention only.  Weights are drawn with a spread of 1 / sqrt(fan-in), larger for what makes scores, so that
a wrong key, a lost state or a swapped stream moves a row by far more than rounding; decays and step sizes are
spread so that some channels forget at once and others keep hundreds of tokens.
"""

import json
import math
import random

import torch

import plain_zifunex as plain
from tinyvllm_b200.models import ZifunexConfig
from tinyvllm_b200.models.zifunex import (ZifunexAttention, ZifunexBigram, ZifunexLayer, ZifunexLinearAttention,
                                          ZifunexLoop, ZifunexScan)


def _p(attention, scan, ff):
    heads, kv, dim, vdim, rot, softcap = attention
    inner, state, rank, taps = scan
    left = ZifunexAttention(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=2.0 / math.sqrt(dim), softcap=softcap,
                            **({} if rot is None else {"rot_dims": rot[0], "rot_base": rot[1]}))
    return ZifunexLayer(left=left, right=ZifunexScan(inner=inner, state=state, dt_rank=rank, conv=taps), ff=ff)


def _g(heads, dim, vdim, tau, ff):
    return ZifunexLayer(linear=ZifunexLinearAttention(heads=heads, dim=dim, vdim=vdim, tau=tau), ff=ff)


ZIFUNEX_CONFIGS = {
    # both mixers, half of a head's dimensions turn, values wider than keys; a loop over the middle run twice; a
    # parallel layer without a feed-forward, a linear one with
    "a": ZifunexConfig(vocab=150, width=64, norm_eps=1e-5, streams=4, bigram=ZifunexBigram(101, 13, 5),
                       loop=ZifunexLoop(1, 3, 2), layers=(
        _p((4, 2, 16, 32, (8, 100.0), 6.0), (96, 16, 8, 4), 96),
        _g(4, 16, 32, 12.0, 80),
        _p((4, 4, 32, 16, (32, 5000.0), 20.0), (48, 8, 4, 4), None),
        _p((4, 2, 16, 32, (8, 100.0), 6.0), (96, 16, 8, 4), 96))),
    # sizes no vector access fits, the linear mixer first: three query heads on one kv head, three taps, a loop over
    # the end run three times
    "b": ZifunexConfig(vocab=97, width=50, norm_eps=1e-6, streams=3, bigram=ZifunexBigram(31, 7, 3),
                       loop=ZifunexLoop(1, 3, 3), layers=(
        _g(3, 10, 7, 5.0, None),
        _p((3, 1, 9, 5, (4, 300.0), 3.0), (37, 7, 5, 3), 30),
        _g(2, 6, 20, 1.0, 22))),
    # a single stream, no loop, as many kv heads as query heads, a scan with one number a channel and one low-rank
    # number, two taps; a wide linear head; no cap
    "c": ZifunexConfig(vocab=130, width=128, norm_eps=1e-6, streams=1, bigram=ZifunexBigram(509, 31, 17), layers=(
        _p((8, 8, 32, 32, (32, 1000000.0), None), (64, 1, 1, 2), 64),
        _g(2, 130, 48, 16.0, None),
        _p((2, 1, 24, 40, None, 1.5), (130, 33, 20, 5), None))),
    # a single head everywhere, one tap, one row of pairs beside the first tokens' row, a loop over everything run
    # once, a state of 20 in as many channels as a warp has lanes less one
    "d": ZifunexConfig(vocab=61, width=36, norm_eps=1e-5, streams=2, bigram=ZifunexBigram(1, 3, 2),
                       loop=ZifunexLoop(0, 2, 1), layers=(
        _p((1, 1, 7, 7, (2, 3.0), 10.0), (31, 20, 3, 1), 20),
        _g(1, 5, 3, 3.0, 12))),
    # sizes of the usual kind (powers of two, heads of 64), four query heads a kv head, a loop over the start
    "e": ZifunexConfig(vocab=300, width=256, norm_eps=1e-6, streams=4, bigram=ZifunexBigram(1021, 127, 7),
                       loop=ZifunexLoop(0, 2, 2), layers=(
        _p((8, 2, 64, 64, (64, 10000.0), 30.0), (512, 16, 16, 4), 384),
        _g(4, 64, 128, 16.0, 256),
        _p((8, 2, 64, 64, (32, 10000.0), 50.0), (256, 32, 16, 4), None))),
    # six streams (a number the kernels are not compiled for), nine taps, a state of 40, no pairs
    "f": ZifunexConfig(vocab=90, width=48, norm_eps=1e-5, streams=6, layers=(
        _p((4, 2, 16, 16, (16, 50.0), 8.0), (72, 40, 9, 9), 40),
        _g(3, 8, 8, 8.0, None),
        _p((4, 1, 32, 48, (8, 70.0), 12.0), (40, 12, 8, 8), 40))),
    # linear attention only: no layer keeps keys or values, a request's whole memory is its state slots
    "g": ZifunexConfig(vocab=90, width=64, norm_eps=1e-5, streams=2, bigram=ZifunexBigram(67, 5, 11),
                       loop=ZifunexLoop(0, 1, 2), layers=(
        _g(2, 16, 16, 4.0, 48),
        _g(4, 8, 24, 10.0, None))),
}
ZIFUNEX_SEEDS = {"a": 51, "b": 52, "c": 53, "d": 54, "e": 55, "f": 56, "g": 57}
ZIFUNEX_PAGES = {"a": 16, "b": 8, "c": 16, "d": 4, "e": 32, "f": 16, "g": 16}
ZIFUNEX_DECAY_RANKS = {"a": 16, "b": 5, "c": 12, "d": 3, "e": 16, "f": 8, "g": 7}


def tensors_of(config: ZifunexConfig, seed: int, decay_rank: int = 8) -> dict:
    """Checkpoint tensors (float32) of ``config``, drawn from ``seed``; ``decay_rank``: rank of the decays' two-step
    projection, which config.json does not give."""
    g = torch.Generator().manual_seed(seed)

    def matrix(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)

    def around_one(n):
        return 1.0 + 0.3 * (torch.rand(n, generator=g) - 0.5)

    def bias(n, spread=0.3):
        return torch.randn(n, generator=g) * spread

    d, s = config.width, config.streams
    t = {"embed": torch.randn(config.vocab, d, generator=g), "final.norm": around_one(d), "final.norm.b": bias(d, 0.1),
         "head": matrix(config.vocab, d, 2.0)}
    if config.bigram is not None:
        t["bigram"] = torch.randn(config.bigram.buckets + 1, d, generator=g)

    def connection(at):
        # every stream is read, kept and written differently; some mixing leads from each stream to each other
        t[at + ".in"] = (0.4 + torch.rand(s, generator=g)) / s ** 0.5 * torch.where(torch.rand(s, generator=g) < 0.3, -1.0, 1.0)
        t[at + ".mix"] = torch.eye(s) * 0.8 + torch.randn(s, s, generator=g) * 0.3 / s ** 0.5
        t[at + ".out"] = 0.4 + torch.rand(s, generator=g)

    for i, layer in enumerate(config.layers):
        p = f"l{i}."
        t[p + "norm1"], t[p + "norm1.b"] = around_one(d), bias(d, 0.1)
        connection(p + "hc1")
        if layer.linear is not None:
            lin = layer.linear
            per, hv = lin.heads * lin.dim, lin.heads * lin.vdim
            t[p + "mix.q"], t[p + "mix.k"] = matrix(per, d, 1.5), matrix(per, d)
            t[p + "mix.v"], t[p + "mix.g"] = matrix(hv, d), matrix(hv, d)
            t[p + "mix.a1"] = matrix(decay_rank, d)
            t[p + "mix.a2"] = matrix(per, decay_rank)
            # from channels that forget within a few tokens to channels that keep hundreds
            t[p + "mix.a2.b"] = torch.rand(per, generator=g) * 8.0 - 1.0
            t[p + "mix.norm"] = around_one(lin.vdim)
            t[p + "mix.o"] = matrix(d, hv)
        else:
            left, right = layer.left, layer.right
            at = p + "mix.left."
            t[at + "q"], t[at + "q.b"] = matrix(left.heads * left.dim, d, 1.5), bias(left.heads * left.dim)
            t[at + "k"], t[at + "k.b"] = matrix(left.kv_heads * left.dim, d, 1.5), bias(left.kv_heads * left.dim)
            t[at + "v"], t[at + "v.b"] = matrix(left.kv_heads * left.vdim, d), bias(left.kv_heads * left.vdim)
            t[at + "o"], t[at + "o.b"] = matrix(d, left.heads * left.vdim), bias(d)
            t[at + "out"] = around_one(d)
            at, inner, n, rank = p + "mix.right.", right.inner, right.state, right.dt_rank
            t[at + "in"] = matrix(2 * inner, d)
            t[at + "conv"] = torch.randn(inner, right.conv, generator=g) / math.sqrt(right.conv)
            t[at + "conv.b"] = bias(inner)
            t[at + "x"] = matrix(rank + 2 * n, inner, 2.0)
            t[at + "dt"] = matrix(inner, rank, 0.5)
            t[at + "dt.b"] = torch.rand(inner, generator=g) * 5.0 - 5.0
            t[at + "A_log"] = torch.rand(inner, n, generator=g) * 4.0 - 3.0
            t[at + "D"] = around_one(inner)
            t[at + "o"] = matrix(d, inner)
            t[at + "out"] = around_one(d)
        if layer.ff is not None:
            t[p + "norm2"], t[p + "norm2.b"] = around_one(d), bias(d, 0.1)
            connection(p + "hc2")
            t[p + "mlp.gate"], t[p + "mlp.up"] = matrix(layer.ff, d, 2.0), matrix(layer.ff, d, 2.0)
            t[p + "mlp.down"] = matrix(d, layer.ff)
    return t


def write_folder(folder, config: ZifunexConfig, seed: int, decay_rank: int = 8, dtype=torch.float32):
    """config.json and model.safetensors of ``config`` in ``folder``.  The values are rounded to
    bfloat16 whatever ``dtype`` stores them as, so that both number formats run the same model."""
    from safetensors.torch import save_file

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config.to_json(), indent=1), encoding="utf-8")
    tensors = {name: value.to(torch.bfloat16).to(dtype).contiguous()
               for name, value in tensors_of(config, seed, decay_rank).items()}
    save_file(tensors, str(folder / "model.safetensors"))
    return folder


def read_folder(folder):
    from safetensors import safe_open

    config = json.loads((folder / "config.json").read_text(encoding="utf-8"))
    tensors = {}
    with safe_open(str(folder / "model.safetensors"), framework="pt", device="cpu") as f:
        for name in f.keys():
            tensors[name] = f.get_tensor(name)
    return config, tensors


_oracle: dict = {}


def oracle_logits(folder, requests: dict) -> dict:
    """{request: float32 logits [T, V]} of the plain implementation, remembered per folder and tokens."""
    config, tensors = read_folder(folder)
    out = {}
    for rid, tokens in requests.items():
        key = (str(folder), tuple(tokens))
        if key not in _oracle:
            _oracle[key] = plain.forward(config, tensors, tokens).to(torch.float32)
        out[rid] = _oracle[key]
    return out


_greedy: dict = {}


def greedy_oracle(folder, prompt, new_tokens: int) -> list[int]:
    key = (str(folder), tuple(prompt), new_tokens)
    if key not in _greedy:
        config, tensors = read_folder(folder)
        _greedy[key] = plain.greedy(config, tensors, prompt, new_tokens)
    return _greedy[key]


def tokens_of(vocab: int, count: int, seed: int) -> list[int]:
    rng = random.Random(seed)
    return [rng.randrange(vocab) for _ in range(count)]

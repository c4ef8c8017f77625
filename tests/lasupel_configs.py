"""Small Lasupel configurations for the tests, their weights and their oracle.

The configurations differ in everything config.json can say: width, vocabulary, scale of the embedding, number and order
of layers (each mixer comes first somewhere); attention with 1, 2, 3 and 4 query heads a kv head, key and value sizes that
are equal or not, multiples of 16 or odd, rotation over a part of a head, over all of it or none, windows of 1 to 100
tokens, shorter and longer than a page, and none; layers that read an earlier layer's keys through a narrower window, a
wider one and none at all, next to it and further on, several of one layer; recurrent units wider and narrower than the
model, of 1 to 16 blocks of sizes that fit vector accesses or not, 1 to 9 taps; delta rules with 1 to 4 value heads a key
head, key sizes from 5 to 130; dense feed-forwards, experts with and without groups, with limits that cut and that do
not, as many chosen as there are, layers without a feed-forward; a model of recurrent layers only.  Weights are drawn
with a spread of 1 / sqrt(fan-in), so that a wrong key or a lost state moves a row by far more than rounding; decays are
spread so that some channels and heads forget at once and others keep hundreds of tokens.
"""

import json
import math
import random

import torch

import plain_lasupel as plain
from tinyvllm_b200.models import LasupelConfig
from tinyvllm_b200.models.lasupel import (LasupelAttention, LasupelDelta, LasupelFeedForward, LasupelLayer,
                                          LasupelRecurrentUnit)


def _dense(ff):
    return LasupelFeedForward(kind="dense", ff=ff)


def _moe(experts, top, ff, limit, groups=1, keep=1):
    return LasupelFeedForward(kind="moe", ff=ff, limit=limit, experts=experts, top=top, groups=groups, keep=keep)


def _a(heads, kv, dim, vdim, window, rot, mlp, kv_from=None):
    rotation = {} if rot is None else {"rot_dims": rot[0], "rot_base": rot[1]}
    return LasupelLayer(LasupelAttention(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=1.5 / math.sqrt(dim),
                                         window=window, kv_from=kv_from, **rotation), mlp)


def _r(width, blocks, conv, mlp):
    return LasupelLayer(LasupelRecurrentUnit(width=width, blocks=blocks, conv=conv), mlp)


def _d(heads, kv, dim, vdim, conv, mlp):
    return LasupelLayer(LasupelDelta(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv), mlp)


LASUPEL_CONFIGS = {
    # every mixer, experts in groups; the reader's window is wider than that of the layer whose keys it reads, so that
    # pages outlive the narrower one
    "a": LasupelConfig(vocab=150, width=64, norm_eps=1e-5, embedding_scale=2.0, layers=(
        _r(96, 4, 4, _dense(96)),
        _a(4, 2, 16, 32, 24, (8, 100.0), _moe(6, 2, 24, 1.0, 3, 2)),
        _d(4, 2, 16, 32, 4, _moe(6, 2, 24, 1.0, 3, 2)),
        _a(8, 2, 16, 32, 75, (8, 100.0), _dense(80), kv_from=1))),
    # sizes no vector access fits, attention first: three query heads on one kv head, values narrower than keys, a
    # window inside a page; three value heads a key head; as many experts chosen as there are
    "b": LasupelConfig(vocab=97, width=50, norm_eps=1e-6, embedding_scale=0.7, layers=(
        _a(3, 1, 9, 5, 5, (4, 300.0), _dense(30)),
        _r(39, 3, 3, _moe(3, 3, 10, 0.4)),
        _d(3, 1, 10, 7, 2, None),
        _a(3, 1, 9, 5, 3, (4, 300.0), _dense(22), kv_from=0))),
    # the delta rule first, as many kv heads as query heads, one block of gates, a layer that reads all keys of one with
    # a window and another that reads them through the same window; four groups of which two are kept
    "c": LasupelConfig(vocab=130, width=128, norm_eps=1e-6, embedding_scale=1.0, layers=(
        _d(2, 2, 32, 48, 8, _moe(8, 3, 32, 7.0, 4, 2)),
        _a(4, 4, 32, 32, 40, (32, 1000000.0), None),
        _r(64, 1, 2, _dense(64)),
        _a(4, 4, 32, 32, None, (32, 1000000.0), None, kv_from=1),
        _a(8, 4, 32, 32, 40, (32, 1000000.0), _dense(64), kv_from=1))),
    # a single head everywhere, one tap, blocks of one channel, a window of one token (a token sees itself), no rotation
    "d": LasupelConfig(vocab=61, width=36, norm_eps=1e-5, embedding_scale=3.5, layers=(
        _r(31, 31, 1, None),
        _a(1, 1, 7, 7, 1, None, _moe(2, 1, 20, 1.5, 2, 1)),
        _d(1, 1, 5, 3, 1, _dense(12)),
        _a(2, 1, 8, 12, 17, (2, 3.0), None))),
    # sizes of the usual kind (powers of two, heads of 64), four query heads a kv head, two value heads a key head
    "e": LasupelConfig(vocab=300, width=256, norm_eps=1e-6, embedding_scale=16.0, layers=(
        _r(256, 4, 4, _dense(384)),
        _d(4, 2, 64, 128, 4, _dense(256)),
        _a(8, 2, 64, 64, 100, (64, 10000.0), _moe(8, 2, 64, 2.5, 2, 1)),
        _a(8, 2, 64, 64, 60, (64, 10000.0), _dense(256), kv_from=2))),
    # nine taps, sixteen blocks, a key size beyond 128, four value heads a key head
    "f": LasupelConfig(vocab=90, width=48, norm_eps=1e-5, embedding_scale=0.25, layers=(
        _d(4, 1, 130, 24, 9, _moe(5, 2, 16, 0.5)),
        _r(128, 16, 9, _moe(12, 4, 8, 1.0, 6, 5)),
        _a(4, 1, 32, 48, 33, (8, 70.0), _dense(40)))),
    # recurrent layers only: no layer keeps keys or values, a request's whole memory is its state slots
    "g": LasupelConfig(vocab=90, width=64, norm_eps=1e-5, embedding_scale=8.0, layers=(
        _r(64, 2, 4, _dense(48)),
        _d(2, 2, 16, 16, 3, None))),
}
LASUPEL_SEEDS = {"a": 61, "b": 62, "c": 63, "d": 64, "e": 65, "f": 66, "g": 67}
LASUPEL_PAGES = {"a": 16, "b": 8, "c": 16, "d": 4, "e": 32, "f": 16, "g": 16}


def tensors_of(config: LasupelConfig, seed: int) -> dict:
    """Checkpoint tensors (float32) of ``config``, drawn from ``seed``."""
    g = torch.Generator().manual_seed(seed)

    def matrix(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)

    def around_one(n):
        return 1.0 + 0.3 * (torch.rand(n, generator=g) - 0.5)

    def bias(n, spread=0.3):
        return torch.randn(n, generator=g) * spread

    def taps(channels, count):
        return torch.randn(channels, count, generator=g) / math.sqrt(count)

    d = config.width
    # sublayers read the stream as it is: projections of a stream that starts at the embedding's scale are kept in range
    size = max(1.0, config.embedding_scale)
    t = {"embed": torch.randn(config.vocab, d, generator=g), "final.norm": around_one(d), "head": matrix(config.vocab, d, 2.0)}
    for i, layer in enumerate(config.layers):
        p, m = f"l{i}.", layer.mixer
        at = p + "mix."
        t[p + "norm1"] = around_one(d) * size
        if layer.type == "attention":
            t[at + "q"], t[at + "o"] = matrix(m.heads * m.dim, d), matrix(d, m.heads * m.vdim)
            if m.kv_from is None:
                t[at + "k"], t[at + "v"] = matrix(m.kv_heads * m.dim, d), matrix(m.kv_heads * m.vdim, d)
        elif layer.type == "rglru":
            c, block = m.width, m.width // m.blocks
            t[at + "y"], t[at + "y.b"] = matrix(c, d, 1.0 / size), bias(c)
            t[at + "x"], t[at + "x.b"] = matrix(c, d, 1.0 / size), bias(c)
            t[at + "conv"], t[at + "conv.b"] = taps(c, m.conv), bias(c)
            for gate in ("ra", "ri"):
                t[at + gate] = torch.randn(m.blocks, block, block, generator=g) / math.sqrt(block)
                t[at + gate + ".b"] = torch.randn(m.blocks, block, generator=g) * 0.5
            # from channels that forget within a token to channels that keep hundreds
            t[at + "lam"] = torch.rand(c, generator=g) * 9.0 - 8.0
            t[at + "o"] = matrix(d, c)
        else:
            per, hv = m.kv_heads * m.dim, m.heads * m.vdim
            for name, rows in (("q", per), ("k", per), ("v", hv)):
                t[at + name], t[at + name + ".conv"] = matrix(rows, d, 1.0 / size), taps(rows, m.conv)
            t[at + "g"] = matrix(hv, d, 1.0 / size)
            t[at + "b"], t[at + "a"] = matrix(m.heads, d, 2.0 / size), matrix(m.heads, d, 1.0 / size)
            t[at + "A_log"] = torch.linspace(-6.0, 1.0, m.heads) if m.heads > 1 else torch.tensor([-3.0])
            t[at + "dt_bias"] = bias(m.heads, 0.5)
            t[at + "norm"] = around_one(m.vdim)
            t[at + "o"] = matrix(d, hv)
        if layer.mlp is None:
            continue
        t[p + "norm2"] = around_one(d) * size
        at, f = p + "mlp.", layer.mlp
        if f.kind == "dense":
            t[at + "gate"], t[at + "up"], t[at + "down"] = matrix(f.ff, d, 2.0 / size), matrix(f.ff, d, 2.0 / size), matrix(d, f.ff)
        else:
            t[at + "router"] = matrix(f.experts, d, 2.0 / size)
            for e in range(f.experts):
                t[at + f"e{e}.gate"], t[at + f"e{e}.up"] = matrix(f.ff, d, 2.0 / size), matrix(f.ff, d, 2.0 / size)
                t[at + f"e{e}.down"] = matrix(d, f.ff)
    return t


def write_folder(folder, config: LasupelConfig, seed: int, dtype=torch.float32):
    """config.json and model.safetensors of ``config`` in ``folder``.  The values are rounded to
    bfloat16 whatever ``dtype`` stores them as, so that both number formats run the same model."""
    from safetensors.torch import save_file

    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config.to_json(), indent=1), encoding="utf-8")
    tensors = {name: value.to(torch.bfloat16).to(dtype).contiguous() for name, value in tensors_of(config, seed).items()}
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

"""A plain, slow Zifunex on the CPU, one function per mechanism, written from the design's equations.

It shares no code with the package: tensors come as a dict name -> torch tensor, the configuration as
the parsed config.json.  Everything runs in ``dtype`` (float64 by default), a token at a time where
the design is a recurrence, with full score matrices where it is attention.
"""

from __future__ import annotations

import torch


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh((2.0 / torch.pi) ** 0.5 * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def layer_norm(x, w, b, eps):
    """(x - mean) / sqrt(mean squared deviation + eps) * w + b over the last dimension."""
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w + b


# ------------------------------------------------------------------ embedding
def bigram_rows(tokens, bigram, previous=None):
    """The row of the pair table each token reads: a hash of the token before it and itself; a sequence's first
    token (``previous`` None) reads the last row, number ``buckets``."""
    rows = []
    for token in tokens:
        if previous is None:
            rows.append(bigram["buckets"])
        else:
            rows.append((previous * bigram["mul_prev"] + token * bigram["mul_cur"]) % bigram["buckets"])
        previous = token
    return rows


def embed(tokens, w, bigram, previous=None):
    x = w["embed"][list(tokens)]
    return x if bigram is None else x + w["bigram"][bigram_rows(tokens, bigram, previous)]


# ------------------------------------------------------------------ attention
def rotate_halves(x, positions, rot):
    """x [tokens, heads, dim]: dimension i and i + dims / 2 of the first ``dims`` turn together by p * base^(-2i/dims)."""
    half = rot["dims"] // 2
    f = torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(half)], dtype=x.dtype)
    angle = positions.to(x.dtype)[:, None, None] * f
    u, v = x[..., :half], x[..., half:2 * half]
    turned = [u * torch.cos(angle) - v * torch.sin(angle), v * torch.cos(angle) + u * torch.sin(angle)]
    return torch.cat(turned + [x[..., 2 * half:]], dim=-1)


def capped_scores(q, k, scale, softcap):
    """cap * tanh(q . k * scale / cap) of [queries, heads, dim] against [keys, heads, dim]: [heads, queries, keys]."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    return s if softcap is None else softcap * torch.tanh(s / softcap)


def softcapped_attention(h, w, at, mixer):
    """Causal attention with biases on every projection, partial rotation and capped scores."""
    tokens, heads, kv = h.shape[0], mixer["heads"], mixer["kv_heads"]
    q = (h @ w[f"{at}.q"].T + w[f"{at}.q.b"]).view(tokens, heads, mixer["dim"])
    k = (h @ w[f"{at}.k"].T + w[f"{at}.k.b"]).view(tokens, kv, mixer["dim"])
    v = (h @ w[f"{at}.v"].T + w[f"{at}.v.b"]).view(tokens, kv, mixer["vdim"])
    positions = torch.arange(tokens)
    if mixer.get("rot") is not None:
        q, k = rotate_halves(q, positions, mixer["rot"]), rotate_halves(k, positions, mixer["rot"])
    shared = [head // (heads // kv) for head in range(heads)]
    s = capped_scores(q, k[:, shared], mixer["scale"], mixer.get("softcap"))
    s = s.masked_fill(positions[None, None, :] > positions[None, :, None], -torch.inf)
    out = torch.einsum("hij,jhv->ihv", torch.softmax(s, -1), v[:, shared]).reshape(tokens, -1)
    return out @ w[f"{at}.o"].T + w[f"{at}.o.b"]


# ----------------------------------------------------------------- recurrences
def causal_convolution(x, taps, bias, before=None):
    """y[t] = bias + sum_j taps[:, j] * x[t - (K - 1) + j] per channel; ``before`` [K - 1, channels] are the inputs
    ahead of the first token (None: zeros)."""
    k = taps.shape[1]
    before = torch.zeros(k - 1, x.shape[1], dtype=x.dtype) if before is None else before
    padded = torch.cat([before, x])
    y = torch.stack([(padded[t:t + k].T * taps).sum(1) for t in range(x.shape[0])]) + bias
    return y, padded[padded.shape[0] - (k - 1):]


def selective_scan(x, dt, b, c, a, d, state=None):
    """S[ch, n] <- exp(dt A[ch, n]) S[ch, n] + dt x B_n, y = sum_n S[ch, n] C_n + D x, a token at a time."""
    state = torch.zeros_like(a) if state is None else state
    out = []
    for t in range(x.shape[0]):
        state = torch.exp(dt[t][:, None] * a) * state + (dt[t] * x[t])[:, None] * b[t][None, :]
        out.append((state * c[t][None, :]).sum(1) + d * x[t])
    return torch.stack(out), state


def mamba(h, w, at, mixer, state=None, before=None):
    """The selective scan between its projections; returns (output, state, the convolution's last inputs)."""
    inner, n, rank = mixer["inner"], mixer["state"], mixer["dt_rank"]
    xz = h @ w[f"{at}.in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x, tail = causal_convolution(x, w[f"{at}.conv"], w[f"{at}.conv.b"], before)
    x = silu(x)
    p = x @ w[f"{at}.x"].T
    dt = softplus(p[:, :rank] @ w[f"{at}.dt"].T + w[f"{at}.dt.b"])
    y, state = selective_scan(x, dt, p[:, rank:rank + n], p[:, rank + n:], -torch.exp(w[f"{at}.A_log"]), w[f"{at}.D"], state)
    return (y * silu(z)) @ w[f"{at}.o"].T, state, tail


def channel_decays(h, w, at, tau):
    """sigmoid(z)^(1 / tau) of the two-step projection z."""
    return torch.sigmoid((h @ w[f"{at}.a1"].T) @ w[f"{at}.a2"].T + w[f"{at}.a2.b"]) ** (1.0 / tau)


def decayed_linear_attention(q, k, v, alpha, state=None):
    """S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head; q, k, alpha [tokens, heads, dim]."""
    state = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(q.shape[0]):
        state = alpha[t][:, :, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(out), state


def gla(h, w, at, mixer, eps, state=None):
    tokens, heads, dim, vdim = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"]
    q = (h @ w[f"{at}.q"].T).view(tokens, heads, dim) * dim ** -0.5
    k = (h @ w[f"{at}.k"].T).view(tokens, heads, dim)
    v = (h @ w[f"{at}.v"].T).view(tokens, heads, vdim)
    alpha = channel_decays(h, w, at, mixer["tau"]).view(tokens, heads, dim)
    o, state = decayed_linear_attention(q, k, v, alpha, state)
    o = rms_norm(o, w[f"{at}.norm"], eps).reshape(tokens, -1)
    return (o * silu(h @ w[f"{at}.g"].T)) @ w[f"{at}.o"].T, state


# -------------------------------------------------------------------- sublayers
def half_sum_of_normed(left, right, left_w, right_w, eps):
    return 0.5 * (rms_norm(left, left_w, eps) + rms_norm(right, right_w, eps))


def parallel(h, w, at, mixer, eps):
    left = softcapped_attention(h, w, f"{at}.left", mixer["left"])
    right, _, _ = mamba(h, w, f"{at}.right", mixer["right"])
    return half_sum_of_normed(left, right, w[f"{at}.left.out"], w[f"{at}.right.out"], eps)


def feed_forward(h, w, at):
    return (gelu_tanh(h @ w[f"{at}.gate"].T) * (h @ w[f"{at}.up"].T)) @ w[f"{at}.down"].T


def read_streams(streams, w_in):
    """u = sum_s in[s] x_s of streams [tokens, streams, width]."""
    return torch.einsum("s,tsw->tw", w_in, streams)


def write_streams(streams, y, mix, w_out):
    """x_t <- sum_s mix[s, t] x_s + out[t] y, all from the old streams."""
    return torch.einsum("st,nsw->ntw", mix, streams) + w_out[None, :, None] * y[:, None, :]


def run_order(cfg):
    loop = cfg.get("loop")
    count = len(cfg["layers"])
    if not loop:
        return list(range(count))
    inside = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inside * loop["times"] + list(range(loop["stop"], count))


def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [tokens, vocab]; ``layers_out`` (a list) collects the sum of the streams after every layer run."""
    w = {name: t.to(dtype) for name, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, w, cfg.get("embedding", {}).get("bigram"))
    streams = x[:, None, :].repeat(1, cfg["streams"], 1)
    for index in run_order(cfg):
        layer, at = cfg["layers"][index], f"l{index}"

        def norm(u, which):
            return layer_norm(u, w[f"{at}.{which}"], w[f"{at}.{which}.b"], eps)

        h = norm(read_streams(streams, w[f"{at}.hc1.in"]), "norm1")
        if layer["type"] == "parallel":
            y = parallel(h, w, f"{at}.mix", layer["mixer"], eps)
        else:
            y, _ = gla(h, w, f"{at}.mix", layer["mixer"], eps)
        streams = write_streams(streams, y, w[f"{at}.hc1.mix"], w[f"{at}.hc1.out"])
        if layer["mlp"] is not None:
            h = norm(read_streams(streams, w[f"{at}.hc2.in"]), "norm2")
            streams = write_streams(streams, feed_forward(h, w, f"{at}.mlp"), w[f"{at}.hc2.mix"], w[f"{at}.hc2.out"])
        if layers_out is not None:
            layers_out.append(streams.sum(1))
    x = layer_norm(streams.sum(1), w["final.norm"], w["final.norm.b"], eps)
    return x @ w["head"].T


def greedy(cfg, weights, prompt, new_tokens: int) -> list[int]:
    tokens = list(prompt)
    for _ in range(new_tokens):
        tokens.append(int(forward(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]

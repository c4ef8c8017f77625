"""A plain, slow Lasupel on the CPU, one function per mechanism, written from the design's equations.

It shares no code with the package: tensors come as a dict name -> torch tensor, the configuration as
the parsed config.json.  Everything runs in ``dtype`` (float64 by default), a token at a time where
the design is a recurrence, with full score matrices where it is attention.
"""

from __future__ import annotations

import torch

UNIT_EPS = 1e-6            # inside the root of the delta rule's unit vectors
DECAY_POWER = 8.0          # the linear recurrent unit's decay at r = 1 is sigmoid(-lam)^8
EXPERT_ALPHA = 1.702


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh((2.0 / torch.pi) ** 0.5 * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def over_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit(x):
    """x / sqrt(sum(x^2) + 1e-6) over the last dimension."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


# ------------------------------------------------------------------ attention
def rotate_halves(x, positions, rot):
    """x [tokens, heads, dim]: dimension i and i + dims / 2 of the first ``dims`` turn together by p * base^(-2i/dims)."""
    half = rot["dims"] // 2
    f = torch.tensor([float(rot["base"]) ** (-2.0 * i / rot["dims"]) for i in range(half)], dtype=x.dtype)
    angle = positions.to(x.dtype)[:, None, None] * f
    u, v = x[..., :half], x[..., half:2 * half]
    turned = [u * torch.cos(angle) - v * torch.sin(angle), v * torch.cos(angle) + u * torch.sin(angle)]
    return torch.cat(turned + [x[..., 2 * half:]], dim=-1)


def prepared_heads(h, weight, heads, dim, rot, eps, positions):
    """A projection's heads, turned by their positions, then each divided by its root mean square."""
    x = (h @ weight.T).view(h.shape[0], heads, dim)
    if rot is not None:
        x = rotate_halves(x, positions, rot)
    return over_rms(x, eps)


def softmax_with_sink(s):
    """exp(s_j) / (1 + sum exp(s_j)) over the last dimension."""
    top = torch.clamp(s.amax(-1, keepdim=True), min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def visible(queries, keys, window):
    """[queries, keys]: 0 <= i - j < window."""
    apart = queries[:, None] - keys[None, :]
    seen = apart >= 0
    return seen if window is None else seen & (apart < window)


def attend(q, k, v, scale, seen):
    """q [queries, heads, dim] against k, v [keys, kv heads, ...]; query head h reads kv head h // (heads / kv heads)."""
    group = q.shape[1] // k.shape[1]
    shared = [head // group for head in range(q.shape[1])]
    s = torch.einsum("ihd,jhd->hij", q, k[:, shared]) * scale
    p = softmax_with_sink(s.masked_fill(~seen[None], -torch.inf))
    return torch.einsum("hij,jhv->ihv", p, v[:, shared])


def attention(h, w, at, mixer, eps, shared=None):
    """Returns (output, (keys, values)); with ``shared`` keys and values are another layer's."""
    positions = torch.arange(h.shape[0])
    rot = mixer.get("rot")
    q = prepared_heads(h, w[f"{at}.q"], mixer["heads"], mixer["dim"], rot, eps, positions)
    if shared is None:
        k = prepared_heads(h, w[f"{at}.k"], mixer["kv_heads"], mixer["dim"], rot, eps, positions)
        v = (h @ w[f"{at}.v"].T).view(h.shape[0], mixer["kv_heads"], mixer["vdim"])
    else:
        k, v = shared
    window = None if mixer.get("mask") is None else mixer["mask"]["size"]
    out = attend(q, k, v, mixer["scale"], visible(positions, positions, window))
    return out.reshape(h.shape[0], -1) @ w[f"{at}.o"].T, (k, v)


# ----------------------------------------------------------------- recurrences
def causal_convolution(x, taps, before=None):
    """y[t] = sum_j taps[:, j] * x[t - (K - 1) + j] per channel; ``before`` [K - 1, channels] are the inputs ahead of
    the first token (None: zeros).  Returns (y, the last K - 1 inputs)."""
    k = taps.shape[1]
    before = torch.zeros(k - 1, x.shape[1], dtype=x.dtype) if before is None else before
    padded = torch.cat([before, x])
    y = torch.stack([(padded[t:t + k].T * taps).sum(1) for t in range(x.shape[0])])
    return y, padded[padded.shape[0] - (k - 1):]


def block_gate(u, weight, bias):
    """sigmoid(A_b u_b + bias_b), u cut into as many parts as there are square matrices."""
    blocks, size = bias.shape
    parts = u.view(u.shape[0], blocks, size)
    return torch.sigmoid(torch.einsum("tbi,boi->tbo", parts, weight) + bias).reshape(u.shape[0], -1)


def gated_linear_unit_scan(u, r, i, lam, state=None):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam), a channel by itself."""
    state = torch.zeros_like(u[0]) if state is None else state
    out = []
    for t in range(u.shape[0]):
        log_a = -DECAY_POWER * r[t] * softplus(lam)
        state = torch.exp(log_a) * state + torch.sqrt(-torch.expm1(2.0 * log_a)) * i[t] * u[t]
        out.append(state)
    return torch.stack(out), state


def rglru(h, w, at, mixer, state=None, before=None):
    """Returns (output, state, the convolution's last inputs)."""
    y = gelu_tanh(h @ w[f"{at}.y"].T + w[f"{at}.y.b"])
    u, tail = causal_convolution(h @ w[f"{at}.x"].T + w[f"{at}.x.b"], w[f"{at}.conv"], before)
    u = u + w[f"{at}.conv.b"]
    r = block_gate(u, w[f"{at}.ra"], w[f"{at}.ra.b"])
    i = block_gate(u, w[f"{at}.ri"], w[f"{at}.ri.b"])
    s, state = gated_linear_unit_scan(u, r, i, w[f"{at}.lam"], state)
    return (s * y) @ w[f"{at}.o"].T, state, tail


def delta_rule(q, k, v, g, beta, state=None):
    """S <- g S; S <- S + k (beta (v - S^T k))^T; o = S^T q per head; q, k [tokens, heads, dim], v [tokens, heads,
    vdim], g and beta [tokens, heads]."""
    state = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state
    out = []
    for t in range(q.shape[0]):
        state = g[t][:, None, None] * state
        write = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", state, k[t]))
        state = state + k[t][:, :, None] * write[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(out), state


def delta_inputs(h, w, at, mixer, before=None):
    """(q, k, v, g, beta, last inputs of the three convolutions) of the delta rule, a head each."""
    tokens, heads, kv = h.shape[0], mixer["heads"], mixer["kv_heads"]
    before = before or {}
    mixed, tails = {}, {}
    for name in ("q", "k", "v"):
        y, tails[name] = causal_convolution(h @ w[f"{at}.{name}"].T, w[f"{at}.{name}.conv"], before.get(name))
        mixed[name] = silu(y)
    shared = [head // (heads // kv) for head in range(heads)]
    q = unit(mixed["q"].view(tokens, kv, mixer["dim"]))[:, shared] * mixer["dim"] ** -0.5
    k = unit(mixed["k"].view(tokens, kv, mixer["dim"]))[:, shared]
    v = mixed["v"].view(tokens, heads, mixer["vdim"])
    beta = torch.sigmoid(h @ w[f"{at}.b"].T)
    g = torch.exp(-torch.exp(w[f"{at}.A_log"]) * softplus(h @ w[f"{at}.a"].T + w[f"{at}.dt_bias"]))
    return q, k, v, g, beta, tails


def delta(h, w, at, mixer, eps, state=None, before=None):
    """Returns (output, state, last inputs of the convolutions)."""
    q, k, v, g, beta, tails = delta_inputs(h, w, at, mixer, before)
    o, state = delta_rule(q, k, v, g, beta, state)
    o = (over_rms(o, eps) * w[f"{at}.norm"]).reshape(h.shape[0], -1)
    return (o * silu(h @ w[f"{at}.g"].T)) @ w[f"{at}.o"].T, state, tails


# ---------------------------------------------------------------- feed-forward
def dense(h, w, at):
    return (silu(h @ w[f"{at}.gate"].T) * (h @ w[f"{at}.up"].T)) @ w[f"{at}.down"].T


def chosen_weights(z, top, groups):
    """[tokens, experts]: softmax scores of the chosen experts, 0 elsewhere.  Only experts of the groups with the
    largest best score can be chosen."""
    s = torch.softmax(z, -1)
    count, keep = (1, 1) if groups is None else (groups["count"], groups["keep"])
    by_group = s.view(s.shape[0], count, -1)
    best = by_group.amax(-1).topk(keep, -1).indices
    open_ = torch.zeros(s.shape[0], count, dtype=torch.bool).scatter(1, best, True)
    choice = by_group.masked_fill(~open_[..., None], -torch.inf).view_as(s)
    return torch.zeros_like(s).scatter(1, choice.topk(top, -1).indices, 1.0) * s


def expert(h, w, at, limit):
    g = torch.clamp(h @ w[f"{at}.gate"].T, max=limit)
    u = torch.clamp(h @ w[f"{at}.up"].T, -limit, limit)
    return (g * torch.sigmoid(EXPERT_ALPHA * g) * (u + 1.0)) @ w[f"{at}.down"].T


def experts(h, w, at, mlp):
    router = mlp["router"]
    weights = chosen_weights(h @ w[f"{at}.router"].T, router["top"], router.get("groups"))
    return sum(weights[:, e:e + 1] * expert(h, w, f"{at}.e{e}", mlp["expert"]["limit"]) for e in range(router["experts"]))


# ----------------------------------------------------------------------- model
def forward(cfg, weights, tokens, dtype=torch.float64, layers_out=None):
    """Logits [tokens, vocab]; ``layers_out`` (a list) collects the residual stream after every layer."""
    w = {name: t.to(dtype) for name, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][list(tokens)] * cfg["embedding"]["scale"]
    kept = {}
    for index, layer in enumerate(cfg["layers"]):
        at, mixer = f"l{index}", layer["mixer"]
        if layer["type"] == "attention":
            y, kept[index] = attention(x, w, f"{at}.mix", mixer, eps, kept.get(mixer.get("kv_from")))
        elif layer["type"] == "rglru":
            y = rglru(x, w, f"{at}.mix", mixer)[0]
        else:
            y = delta(x, w, f"{at}.mix", mixer, eps)[0]
        x = x + over_rms(y, eps) * w[f"{at}.norm1"]
        mlp = layer.get("mlp")
        if mlp is not None:
            y = dense(x, w, f"{at}.mlp") if mlp["kind"] == "dense" else experts(x, w, f"{at}.mlp", mlp)
            x = x + over_rms(y, eps) * w[f"{at}.norm2"]
        if layers_out is not None:
            layers_out.append(x)
    return (over_rms(x, eps) * w["final.norm"]) @ w["head"].T


def greedy(cfg, weights, prompt, new_tokens: int) -> list[int]:
    tokens = list(prompt)
    for _ in range(new_tokens):
        tokens.append(int(forward(cfg, weights, tokens)[-1].argmax()))
    return tokens[len(prompt):]

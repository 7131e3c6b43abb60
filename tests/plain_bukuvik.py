"""Bukuvik written out plainly: one function per mechanism, 64-bit, whole sequences, no cache, no batch.

The yardstick of the Bukuvik tests. It shares no code with the engine: it reads a configuration dict and a dict of stored
tensors and walks a sequence's tokens with loops and small matrix products. Notation: x a token's row of the stream, W y a
stored weight [out, in] applied to y, R(y) = y / sqrt(mean(y²) + eps).

    stream:     x = s · embed[token];  x ← x + m · a1 ∘ w1 ∘ R(mixer(x));  x ← x + m · a2 ∘ w2 ∘ R(ff(x)); the sublayers read x;
                logits = embed · (w ∘ R(x))
    two maps:   attention with two sets of queries and keys and one of values; each set makes its own softmax over the keys
                of a window; a head's output is R(o1 − λ o2) · (1 − d), λ = exp(Σ lq1 lk1) − exp(Σ lq2 lk2) + d
    side by side: ½ (w_l ∘ R(left(x)) + w_r ∘ R(right(x)))
      left:     attention over a window that also keeps the sequence's first tokens; q and k turned, then divided by their
                root mean square; heads gated by sigmoid(W_g x)
      right:    a state S [N, V] per head: S ← exp(−e^A dt) S + dt B xᵀ, y = Sᵀ C + D x, dt = softplus(· + bias); x, B, C
                through a short convolution and silu; y · silu(z) normed in equal parts
    ff:         W_down relu(W_up x)²
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def _w(weights, name):
    return weights[name].to(F)


def unit_rms(y, eps):
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)


def frequencies(rot):
    """(frequency of every turned pair, the factor on cosines and sines)."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    pair_of = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))      # noqa: E731
    lo, hi = max(math.floor(pair_of(s["fast"])), 0), min(math.ceil(pair_of(s["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * r + x * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def turn_halves(x, positions, rot):
    """x [t, ..., dim]: channels (i, i + dims / 2), i < dims / 2, turned by position · frequency."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    f, size = frequencies(rot)
    angle = positions.to(F)[:, None] * torch.tensor(f, dtype=F)[None]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (half,)
    cos, sin = (angle.cos() * size).view(shape), (angle.sin() * size).view(shape)
    a, b = x[..., :half], x[..., half:2 * half]
    return torch.cat((a * cos - b * sin, b * cos + a * sin, x[..., 2 * half:]), dim=-1)


def visible(i, j, mask):
    """Whether position i sees position j."""
    if j > i:
        return False
    size = mask["size"] if mask else 0
    return not size or i - j < size or j < (mask.get("keep_first") or 0)


def attend(q, k, v, scale, mask, cap=None):
    """q, k [t, dim], v [t, vdim] of one head -> [t, vdim]."""
    t = q.shape[0]
    s = (q @ k.T) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    hidden = torch.tensor([[not visible(i, j, mask) for j in range(t)] for i in range(t)])
    return torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v


def two_map_attention(x, weights, p, m, eps):
    t = x.shape[0]
    heads, kvh, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (x @ _w(weights, p + "q").T).view(t, heads, 2, dim)
    k = (x @ _w(weights, p + "k").T).view(t, kvh, 2, dim)
    v = (x @ _w(weights, p + "v").T).view(t, kvh, vdim)
    pos = torch.arange(t)
    q = turn_halves(unit_rms(q, eps) * _w(weights, p + "q.norm"), pos, m.get("rot"))
    k = turn_halves(unit_rms(k, eps) * _w(weights, p + "k.norm"), pos, m.get("rot"))
    d = float(m["diff"])
    lam = math.exp(float(_w(weights, p + "lq1") @ _w(weights, p + "lk1"))) \
        - math.exp(float(_w(weights, p + "lq2") @ _w(weights, p + "lk2"))) + d
    out = torch.zeros(t, heads, vdim, dtype=F)
    for h in range(heads):
        g = h // (heads // kvh)
        one, two = (attend(q[:, h, i], k[:, g, i], v[:, g], m["scale"], m.get("mask"), m.get("softcap")) for i in (0, 1))
        out[:, h] = unit_rms(one - lam * two, eps) * (1.0 - d)
    y = out.reshape(t, heads * vdim) * torch.sigmoid(x @ _w(weights, p + "g").T)
    return y @ _w(weights, p + "o").T


def kept_window_attention(x, weights, p, m, eps):
    t = x.shape[0]
    heads, kvh, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(t)
    q = unit_rms(turn_halves((x @ _w(weights, p + "q").T).view(t, heads, dim), pos, m.get("rot")), eps)
    k = unit_rms(turn_halves((x @ _w(weights, p + "k").T).view(t, kvh, dim), pos, m.get("rot")), eps)
    v = (x @ _w(weights, p + "v").T).view(t, kvh, vdim)
    out = torch.stack([attend(q[:, h], k[:, h // (heads // kvh)], v[:, h // (heads // kvh)], m["scale"], m.get("mask"))
                       for h in range(heads)], dim=1)
    y = out.reshape(t, heads * vdim) * torch.sigmoid(x @ _w(weights, p + "g").T)
    return y @ _w(weights, p + "o").T


def causal_conv(x, w, b):
    """x [t, channels], w [channels, taps]: the last tap weighs the token itself; zeros before the first token."""
    t, taps = x.shape[0], w.shape[1]
    padded = torch.cat((torch.zeros(taps - 1, x.shape[1], dtype=F), x), 0)
    return sum(padded[j:j + t] * w[:, j] for j in range(taps)) + b


def state_space(x, weights, p, m, eps):
    t = x.shape[0]
    heads, groups, n, vdim = m["heads"], m["groups"], m["state"], m["vdim"]
    inner = heads * vdim
    z, xbc, dt = (x @ _w(weights, p + "in").T).split([inner, inner + 2 * groups * n, heads], -1)
    xbc = torch.nn.functional.silu(causal_conv(xbc, _w(weights, p + "conv"), _w(weights, p + "conv.b")))
    xs, b, c = xbc.split([inner, groups * n, groups * n], -1)
    xs, b, c = xs.reshape(t, heads, vdim), b.reshape(t, groups, n), c.reshape(t, groups, n)
    dt = torch.nn.functional.softplus(dt + _w(weights, p + "dt_bias"), threshold=1e9)
    rate, skip = torch.exp(_w(weights, p + "A_log")), _w(weights, p + "D")
    y = torch.zeros(t, heads, vdim, dtype=F)
    for h in range(heads):
        g = h // (heads // groups)
        S = torch.zeros(n, vdim, dtype=F)
        for i in range(t):
            S = torch.exp(-rate[h] * dt[i, h]) * S + dt[i, h] * torch.outer(b[i, g], xs[i, h])
            y[i, h] = S.T @ c[i, g] + skip[h] * xs[i, h]
    y = y.reshape(t, inner) * torch.nn.functional.silu(z)
    y = unit_rms(y.view(t, m["norm_groups"], -1), eps).reshape(t, inner) * _w(weights, p + "norm")
    return y @ _w(weights, p + "o").T


def side_by_side(x, weights, p, m, eps):
    left = unit_rms(kept_window_attention(x, weights, p + "left.", m["left"], eps), eps) * _w(weights, p + "left.out")
    right = unit_rms(state_space(x, weights, p + "right.", m["right"], eps), eps) * _w(weights, p + "right.out")
    return 0.5 * (left + right)


def dense_ff(x, weights, p):
    return torch.relu(x @ _w(weights, p + "up").T) ** 2 @ _w(weights, p + "down").T


MIXERS = {"attention": two_map_attention, "parallel": side_by_side}


def forward(weights, config, ids, streams=None):
    """Logits [tokens, vocab] of one sequence; `streams`, a list, receives the stream behind every layer."""
    eps, mult = float(config["norm"]["eps"]), float(config["residual_mult"])
    table = _w(weights, "embed")
    x = table[torch.tensor(list(ids))] * float(config["embedding"]["scale"])
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](x, weights, p + "mix.", layer["mixer"], eps)
        x = x + mult * unit_rms(y, eps) * _w(weights, p + "norm1") * _w(weights, p + "ls1")
        if layer.get("mlp") is not None:
            y = dense_ff(x, weights, p + "mlp.")
            x = x + mult * unit_rms(y, eps) * _w(weights, p + "norm2") * _w(weights, p + "ls2")
        if streams is not None:
            streams.append(x)
    return unit_rms(x, eps) * _w(weights, "final.norm") @ table.T

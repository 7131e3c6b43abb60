"""Gegunex written out plainly: one function per mechanism, 64-bit, whole sequences, no cache, no batch.

The yardstick of the Gegunex tests. It shares no code with the engine: it reads a configuration dict and a dict of
stored tensors and walks a sequence's tokens with loops and small matrix products. Notation: x a token's row of the
stream, W y a stored weight [out, in] applied to y, N a layer norm, R an RMS norm, rms(y) = sqrt(mean(y²) + eps).

    layer:      x ← x + μ · mixer(N1(x));  x ← x + μ · ff(N2(x)),  N(y) = (y − mean y) / sqrt(var y + eps) · w
    linear:     per head a matrix S: S ← d_h S + k vᵀ, o = Sᵀ q, with q, k, v = silu(W y) and one fixed decay d_h a head;
                all heads' o together: R(o) · weight · sigmoid(W_g y), then W_o
    latent:     q = W_uq R(W_dq y) per head [plain | turned]; W_dkv y = [c' | k'] with c = R(c'), k_r = k' turned, shared by
                the heads; keys W_uk c, values W_uv c per head; score (q_p · k_p + q_r · k_r) · scale over the last
                `mask.size` positions; a softmax whose denominator also holds exp(sink_h); W_o
    delta:      q, k, v through a causal convolution over time and silu; q, k unit vectors per head (q · dim^(−1/2)); a decay per
                key channel g = exp(−exp(A) softplus(W_a2 W_a1 y + bias)), β = sigmoid(W_b y);
                S ← diag(g) S;  S ← S + k (β (v − Sᵀk))ᵀ;  o = Sᵀ q;  R(o) per head · weight · sigmoid(W_g2 W_g1 y); W_o
    experts:    scores s = sigmoid(W_router y); the `top` largest; Σ expert_e(s_e · y);
                expert(y) = W_down (g sigmoid(1.702 g) (u + 1)), g = min(W_gate y, limit), u = W_up y held in ±limit
    head:       cap · tanh(E N(x) / cap) with the embedding table E
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def _w(weights, name):
    return weights[name].to(F)


def layer_norm(y, w, eps):
    d = y - y.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms_norm(y, w, eps):
    return y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z * torch.sigmoid(z)


# ---------------------------------------------------------------- rotation
def frequencies(rot):
    """(angle per position of every pair, factor on cosine and sine)."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def dim(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim(float(scaling["fast"]))), 0)
    hi = min(math.ceil(dim(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(factor) + 1


def turn_neighbours(x, positions, rot):
    """x [t, heads, d]: channels (2i, 2i + 1) of the first rot.dims turned by position · f_i."""
    dims = rot["dims"]
    f, m = frequencies(rot)
    angle = positions.to(F)[:, None] * torch.tensor(f, dtype=F)[None, :]
    cos, sin = (angle.cos() * m)[:, None, :], (angle.sin() * m)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = u * cos - v * sin, v * cos + u * sin
    return out


# ---------------------------------------------------------------- mixers
def linear_state(h, weights, p, m, eps):
    t = h.shape[0]
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ _w(weights, p + "q").T).view(t, heads, dim)
    k = silu(h @ _w(weights, p + "k").T).view(t, heads, dim)
    v = silu(h @ _w(weights, p + "v").T).view(t, heads, vdim)
    out = torch.zeros(t, heads, vdim, dtype=F)
    for g in range(heads):
        S = torch.zeros(dim, vdim, dtype=F)
        for s in range(t):
            S = float(m["decay"][g]) * S + torch.outer(k[s, g], v[s, g])
            out[s, g] = S.T @ q[s, g]
    y = rms_norm(out.reshape(t, heads * vdim), _w(weights, p + "norm"), eps)
    return (y * torch.sigmoid(h @ _w(weights, p + "g").T)) @ _w(weights, p + "o").T


def latent_scores(h, weights, p, m, eps):
    """(scores [heads, query, key] times the scale, unmasked; the latents c)."""
    t = h.shape[0]
    heads, dim, rot, rank = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    pos = torch.arange(t)
    q = (rms_norm(h @ _w(weights, p + "dq").T, _w(weights, p + "dq.norm"), eps) @ _w(weights, p + "uq").T).view(t, heads, dim + rot)
    down = h @ _w(weights, p + "dkv").T
    c = rms_norm(down[:, :rank], _w(weights, p + "dkv.norm"), eps)
    k_r = turn_neighbours(down[:, None, rank:], pos, m["rot"])[:, 0]
    q_r = turn_neighbours(q[:, :, dim:], pos, m["rot"])
    k_p = (c @ _w(weights, p + "uk").T).view(t, heads, dim)
    s = torch.einsum("qhd,khd->hqk", q[:, :, :dim], k_p) + torch.einsum("qhd,kd->hqk", q_r, k_r)
    return s * float(m["scale"]), c


def seen(t, m):
    """[query, key]: True where the query sees the key."""
    back = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return (back >= 0) & (back < m["mask"]["size"])


def latent_attention(h, weights, p, m, eps):
    t = h.shape[0]
    heads, vdim = m["heads"], m["vdim"]
    s, c = latent_scores(h, weights, p, m, eps)
    v = (c @ _w(weights, p + "uv").T).view(t, heads, vdim)
    s = s.masked_fill(~seen(t, m), -math.inf)
    sink = _w(weights, p + "sink")
    top = torch.maximum(s.max(-1).values, sink[:, None])                     # (subtracted above and below the line alike)
    e = torch.exp(s - top[..., None])
    prob = e / (e.sum(-1) + torch.exp(sink[:, None] - top))[..., None]
    return torch.einsum("hqk,khd->qhd", prob, v).reshape(t, heads * vdim) @ _w(weights, p + "o").T


def convolve(x, taps):
    """Per channel over time: y_t = Σ_j taps[c, j] x_(t − (n − 1 − j)), zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat((torch.zeros(n - 1, x.shape[1], dtype=F), x), 0)
    return sum(padded[j:j + x.shape[0]] * taps[:, j] for j in range(n))


def channel_delta(h, weights, p, m, eps):
    t = h.shape[0]
    heads, kvh, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(convolve(h @ _w(weights, p + x).T, _w(weights, f"{p}{x}.conv"))) for x in "qkv")
    q, k, v = q.view(t, kvh, dim), k.view(t, kvh, dim), v.view(t, heads, vdim)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * dim ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = torch.sigmoid(h @ _w(weights, p + "b").T)
    a = (h @ _w(weights, p + "a1").T) @ _w(weights, p + "a2").T + _w(weights, p + "dt_bias")
    rate = torch.exp(_w(weights, p + "A_log"))
    g = torch.exp(-rate[None, :, None] * torch.log1p(torch.exp(a)).view(t, heads, dim))
    out = torch.zeros(t, heads, vdim, dtype=F)
    for e in range(heads):
        kh = e // (heads // kvh)
        S = torch.zeros(dim, vdim, dtype=F)
        for s in range(t):
            S = g[s, e][:, None] * S
            S = S + torch.outer(k[s, kh], beta[s, e] * (v[s, e] - S.T @ k[s, kh]))
            out[s, e] = S.T @ q[s, kh]
    gate = torch.sigmoid((h @ _w(weights, p + "g1").T) @ _w(weights, p + "g2").T)
    y = rms_norm(out, _w(weights, p + "norm"), eps).reshape(t, heads * vdim) * gate
    return y @ _w(weights, p + "o").T


# ---------------------------------------------------------------- feed-forward
def clamped_unit(y, weights, p, limit):
    g = torch.clamp(y @ _w(weights, p + "gate").T, max=limit)
    u = torch.clamp(y @ _w(weights, p + "up").T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ _w(weights, p + "down").T


def choose(z, top):
    """For one token's router logits z: [(expert, weight)]."""
    s = torch.sigmoid(z)
    return [(e, s[e]) for e in torch.topk(z, top).indices.tolist()]


def experts_ff(y, weights, p, mlp):
    z = y @ _w(weights, p + "router").T
    out = torch.zeros_like(y)
    for t in range(y.shape[0]):
        for e, share in choose(z[t], mlp["router"]["top"]):
            out[t] += clamped_unit(share * y[t], weights, f"{p}e{e}.", float(mlp["expert"]["limit"]))
    return out


MIXERS = {"lightning": linear_state, "latent_attention": latent_attention, "channel_delta": channel_delta}


def forward(weights, config, ids, streams=None):
    """Logits [tokens, vocab] of one sequence; `streams`, a list, receives the stream after every layer."""
    eps, mult, cap = float(config["norm"]["eps"]), float(config["residual_mult"]), float(config["logit_softcap"])
    x = _w(weights, "embed")[torch.tensor(list(ids))]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + mult * MIXERS[layer["type"]](layer_norm(x, _w(weights, p + "norm1"), eps), weights, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + mult * experts_ff(layer_norm(x, _w(weights, p + "norm2"), eps), weights, p + "mlp.", layer["mlp"])
        if streams is not None:
            streams.append(x)
    logits = layer_norm(x, _w(weights, "final.norm"), eps) @ _w(weights, "embed").T
    return cap * torch.tanh(logits / cap)

"""Tiny Gegunex configurations, model folders with weights that make faults show, and the comparison with the plain
implementation (tests/plain_gegunex.py) that the CPU and GPU tests of this design share."""
from __future__ import annotations

import json

from safetensors.torch import load_file, save_file
import torch

import plain_gegunex as plain


def _lin(heads, dim, vdim, decay=None):
    decay = decay or [1 - 2.0 ** (-1 - 2 * (h % 4)) for h in range(heads)]
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}


def _lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, sharpen, base=300.0, scaling=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
            "mask": {"size": window}, "scale": sharpen / (dim + rot_dim) ** 0.5, "rot": rot}


def _delta(heads, kv_heads, dim, vdim, taps, decay_rank, gate_rank):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps, "decay_rank": decay_rank,
            "gate_rank": gate_rank}


def _moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def _layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _model(width, vocab, eps, mult, cap, layers):
    return json.loads(json.dumps({"architecture": "Gegunex", "width": width, "vocab": vocab, "norm": {"eps": eps},
                                  "residual_mult": mult, "logit_softcap": cap, "layers": layers}))


# A: the three mixers in turn, two latent layers with windows, ranks and frequencies of their own (one with YaRN, one
# without), a delta rule with two value heads a key head, key and value sizes that differ, several experts a token, a layer
# without a feed-forward.
GA = _model(64, 211, 1e-5, 0.6, 9.0, [
    _layer("channel_delta", _delta(4, 2, 16, 24, 3, 6, 5), _moe(5, 2, 40, 1.5)),
    _layer("latent_attention", _lat(3, 20, 12, 28, 40, 24, 7, 4.0, 300.0, (4.0, 64, 8.0, 1.0)), _moe(6, 3, 24, 0.8)),
    _layer("lightning", _lin(3, 16, 20), _moe(3, 1, 36, 2.0)),
    _layer("latent_attention", _lat(5, 8, 16, 12, 32, 48, 30, 4.0, 10000.0), _moe(4, 4, 16, 1.0)),
    _layer("channel_delta", _delta(2, 2, 8, 8, 4, 4, 4), None)])
# B: sizes that are multiples of nothing, an odd vocabulary, no carried convolution inputs (one tap), three value heads a key
# head, windows of one and of two tokens, a residual multiplier above 1, one expert in all.
GB = _model(72, 157, 1e-6, 1.3, 30.0, [
    _layer("latent_attention", _lat(2, 12, 6, 10, 22, 20, 1, 3.0), _moe(3, 2, 20, 7.0)),
    _layer("channel_delta", _delta(3, 1, 20, 12, 1, 3, 7), _moe(1, 1, 28, 0.5)),
    _layer("lightning", _lin(1, 12, 36, [0.9]), None),
    _layer("latent_attention", _lat(3, 10, 2, 14, 18, 36, 2, 3.0, 50.0, (2.0, 32, 4.0, 0.5)), _moe(7, 5, 12, 1.0))])
# C: sizes the tensor-core kernels take (latents of 32 and 144, rotated parts of 16 and 32), a window longer than a page and one
# that ends inside it, larger heads in the matrix states, a norm over 640 channels, widths of the 8-row expert kernel.
GC = _model(128, 300, 1e-5, 0.5, 20.0, [
    _layer("lightning", _lin(4, 80, 160), _moe(4, 4, 48, 1.2)),
    _layer("latent_attention", _lat(8, 24, 16, 40, 64, 32, 33, 3.0, 1e5, (16.0, 128, 16.0, 2.0)), _moe(5, 3, 64, 1.0)),
    _layer("channel_delta", _delta(2, 1, 96, 32, 4, 16, 12), _moe(2, 2, 32, 3.0)),
    _layer("latent_attention", _lat(4, 32, 32, 32, 48, 144, 90, 3.0, 1e4), _moe(6, 2, 80, 1.0))])
# One mechanism alone.
G_LAT = _model(48, 97, 1e-5, 1.0, 12.0, [_layer("latent_attention", _lat(4, 16, 16, 20, 24, 32, 25, 3.0, 100.0, (3.0, 40, 6.0, 1.0)), None)])
G_LIN = _model(48, 97, 1e-5, 0.8, 12.0, [_layer("lightning", _lin(3, 12, 20), None)])
G_DELTA = _model(48, 97, 1e-5, 0.8, 12.0, [_layer("channel_delta", _delta(4, 2, 16, 12, 4, 6, 5), None)])
G_MOE = _model(48, 97, 1e-5, 0.8, 12.0, [_layer("lightning", _lin(1, 4, 4), _moe(9, 3, 16, 0.7))])
CONFIGS = {"a": GA, "b": GB, "c": GC, "lat": G_LAT, "lin": G_LIN, "delta": G_DELTA, "moe": G_MOE}


def tensor_table(config):
    """(stored name, shape) of every tensor of a model folder, from the configuration alone."""
    w = config["width"]
    out = [("embed", (config["vocab"], w)), ("final.norm", (w,))]
    for i, layer in enumerate(config["layers"]):
        m, mlp, p, x = layer["mixer"], layer.get("mlp"), f"l{i}.", f"l{i}.mix."
        out.append((p + "norm1", (w,)))
        if layer["type"] == "lightning":
            nq, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out += [(x + "q", (nq, w)), (x + "k", (nq, w)), (x + "v", (nv, w)), (x + "g", (nv, w)), (x + "norm", (nv,)), (x + "o", (w, nv))]
        elif layer["type"] == "latent_attention":
            h, rank = m["heads"], m["kv_rank"]
            out += [(x + "dq", (m["q_rank"], w)), (x + "dq.norm", (m["q_rank"],)), (x + "uq", (h * (m["dim"] + m["rot_dim"]), m["q_rank"])),
                    (x + "dkv", (rank + m["rot_dim"], w)), (x + "dkv.norm", (rank,)), (x + "uk", (h * m["dim"], rank)),
                    (x + "uv", (h * m["vdim"], rank)), (x + "sink", (h,)), (x + "o", (w, h * m["vdim"]))]
        else:
            nq, nv, nk = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"] * m["dim"]
            for name, n in (("q", nq), ("k", nq), ("v", nv)):
                out += [(x + name, (n, w)), (x + name + ".conv", (n, m["conv"]))]
            out += [(x + "b", (m["heads"], w)), (x + "A_log", (m["heads"],)), (x + "norm", (m["vdim"],)),
                    (x + "a1", (m["decay_rank"], w)), (x + "a2", (nk, m["decay_rank"])), (x + "dt_bias", (nk,)),
                    (x + "g1", (m["gate_rank"], w)), (x + "g2", (nv, m["gate_rank"])), (x + "o", (w, nv))]
        if mlp is not None:
            out += [(p + "norm2", (w,)), (p + "mlp.router", (mlp["router"]["experts"], w))]
            for e in range(mlp["router"]["experts"]):
                ff = mlp["expert"]["ff"]
                out += [(f"{p}mlp.e{e}.gate", (ff, w)), (f"{p}mlp.e{e}.up", (ff, w)), (f"{p}mlp.e{e}.down", (w, ff))]
    return out


def make_weights(config, seed: int):
    """Random weights, rounded to bfloat16 (so that both sides read the same numbers). Products' weights are N(0, 1/in), so
    activations keep unit size; with the configurations' score scales the attention's scores spread over several units: a
    wrong key, page or window edge moves the logits. Sinks are of the scores' own size (they take a visible share of the
    denominator), routers are spread (scores from near 0 to near 1, so a weight on the wrong side of the expert shows in the
    clamped unit), decay rates are spread so that some channels forget within a few tokens and others keep what the first
    tokens wrote, embeddings carry an offset (a norm that forgets the mean shows)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_table(config):
        x = torch.randn(shape, generator=g, dtype=torch.float32)
        tail = name.split(".", 1)[1] if name.startswith("l") else name
        if name == "embed":
            x = 0.5 + x
        elif tail.endswith(".conv"):
            x = 0.6 * x
        elif tail == "mix.A_log":
            x = -1.0 + 1.5 * x
        elif tail == "mix.sink":
            x = 1.5 + 1.5 * x
        elif tail == "mix.dt_bias":
            pass
        elif len(shape) == 1:
            x = 1.0 + 0.2 * x
        elif tail == "mlp.router":
            x = 2.0 * x / shape[1] ** 0.5
        elif tail.endswith((".gate", ".up")):
            x = 1.5 * x / shape[1] ** 0.5
        else:
            x = x / shape[1] ** 0.5
        out[name] = x.to(torch.bfloat16).contiguous()
    return out


def stored_config(config):
    """The configuration as a model folder stores it: without the two ranks that only tensor shapes give."""
    c = json.loads(json.dumps(config))
    for layer in c["layers"]:
        for key in ("decay_rank", "gate_rank"):
            layer["mixer"].pop(key, None)
    return c


def make_folder(tmp_path, name: str, seed: int = 0, config=None, weights=None):
    config = config or CONFIGS[name]
    folder = tmp_path / f"gegunex_{name}"
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(stored_config(config)))
    save_file(weights if weights is not None else make_weights(config, seed), str(folder / "model.safetensors"))
    return folder


def read_folder(folder):
    import pathlib
    folder = pathlib.Path(folder)
    return json.loads((folder / "config.json").read_text()), load_file(str(folder / "model.safetensors"))


def exact_logits(folder, ids):
    config, weights = read_folder(folder)
    return plain.forward(weights, config, list(ids)).float()


def point_at(config, weights, layer: int, ids, reads: int, key: int, sharp: float):
    """A latent layer's weights changed so that in a model whose FIRST layer it is, the query at position `reads` finds the
    key at position `key` by far the best among all earlier ones in every head, if its window reaches it: W_uk's part is
    built from the two tokens' own latents. Returns new weights; the tokens at both places must be unlike all others."""
    m, p = config["layers"][layer]["mixer"], f"l{layer}.mix."
    out = {k: v.clone() for k, v in weights.items()}
    eps = float(config["norm"]["eps"])
    x = plain.layer_norm(plain._w(weights, "embed")[torch.tensor(list(ids))], plain._w(weights, f"l{layer}.norm1"), eps)
    q = plain.rms_norm(x @ plain._w(weights, p + "dq").T, plain._w(weights, p + "dq.norm"), eps) @ plain._w(weights, p + "uq").T
    q = q.view(len(ids), m["heads"], m["dim"] + m["rot_dim"])[reads, :, :m["dim"]]
    c = plain.rms_norm((x @ plain._w(weights, p + "dkv").T)[:, :m["kv_rank"]], plain._w(weights, p + "dkv.norm"), eps)[key]
    uk = plain._w(weights, p + "uk").view(m["heads"], m["dim"], m["kv_rank"])
    for h in range(m["heads"]):                     # a rank-one part that makes q · W_uk c large for this pair of tokens
        uk[h] += sharp / float(m["scale"]) * torch.outer(q[h] / (q[h] @ q[h]), c / (c @ c))
    out[p + "uk"] = uk.reshape(m["heads"] * m["dim"], m["kv_rank"]).to(torch.bfloat16)
    return out


# The measure, per row: the distance from the plain implementation's 64-bit logits (mean taken off, root mean square over
# the vocabulary) relative to the row's own spread. float32: every row within 2e-4. bfloat16: rounding alone leaves most rows
# 0.005 to 0.04 away; scores are sharp on purpose and routers choose among few experts, so here and there a row turns on a
# close call (another expert of nearly the same score, whose output is another) and lands further off, in the plain twins of the
# kernels just as on the GPU: up to 0.9. So: the median within 0.03, at most one row in fifteen beyond 0.12, none beyond 1.2. A wrong key, state, slot or weight moves every row it touches by a good
# part of its spread, and in 32-bit, where the same schedules run, nothing is excused.
LIMITS = {"float32": 2e-4, "bfloat16": 0.12}


def row_error(got, want):
    d = got.double() - want.double()
    d = d - d.mean()
    spread = (want.double() - want.double().mean()).pow(2).mean().sqrt()
    return float(d.pow(2).mean().sqrt() / spread)


def compare(got, want, dtype):
    """`got`: {(request, position): logits row}; `want`: {request: exact logits [tokens, vocab]}."""
    assert got, "nothing to compare"
    errors = sorted((row_error(row, want[rid][pos]), rid, pos) for (rid, pos), row in got.items())
    worst = errors[-1]
    if dtype == "bfloat16":
        assert worst[0] <= 1.2, f"request {worst[1]} position {worst[2]}: error {worst[0]:.3g} of the row's spread"
        over = [e for e in errors if e[0] > LIMITS[dtype]]
        assert len(over) <= max(1, len(errors) // 15), f"{len(over)} of {len(errors)} rows are beyond {LIMITS[dtype]}: {over[-5:]}"
        assert errors[len(errors) // 2][0] <= 0.03, f"the median row is {errors[len(errors) // 2][0]:.3g} of its spread off"
        return
    assert worst[0] <= LIMITS[dtype], f"request {worst[1]} position {worst[2]}: error {worst[0]:.3g} of the row's spread"

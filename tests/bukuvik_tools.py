"""Tiny Bukuvik configurations, model folders with weights that make faults show, and the comparison with the plain implementation
(tests/plain_bukuvik.py) that the CPU and GPU tests of this design share."""
from __future__ import annotations

import json

import torch
from safetensors.torch import load_file, save_file

import plain_bukuvik as plain


def _rot(base, dims, scaling=None):
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return rot


def _att(heads, kv_heads, dim, vdim, sharpen, size=0, keep=None, rot=None, cap=None, diff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": sharpen / dim ** 0.5}
    if size:
        m["mask"] = {"size": size} if keep is None else {"size": size, "keep_first": keep}
    if rot:
        m["rot"] = rot
    if cap:
        m["softcap"] = cap
    if diff is not None:
        m["diff"] = diff
    return m


def _ssm(heads, groups, state, vdim, taps, norm_groups):
    return {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": taps, "norm_groups": norm_groups}


def _diff(mixer, ff):
    return {"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _par(left, right, ff):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _model(width, vocab, eps, mult, scale, layers):
    return json.loads(json.dumps({"architecture": "Bukuvik", "width": width, "vocab": vocab, "norm": {"eps": eps},
                                  "residual_mult": mult, "embedding": {"scale": scale}, "layers": layers}))


# A: both layer types in turn; windows of 10 and 7 over pages of 4, kept first tokens that end inside a page, a cap that bends the
# scores, rotations of a part of the channels, YaRN, four heads on two, unequal key and value sizes, a layer without feed-forward.
BA = _model(64, 211, 1e-5, 0.7, 2.5, [
    _diff(_att(4, 2, 12, 20, 3.0, 10, rot=_rot(500.0, 8), cap=6.0, diff=0.4), 96),
    _par(_att(4, 2, 16, 12, 4.0, 7, 6, _rot(300.0, 12, (4.0, 64, 8.0, 1.0))), _ssm(6, 2, 10, 8, 3, 3), 72),
    _par(_att(4, 1, 16, 24, 4.0, 12, 3, _rot(1000.0, 16)), _ssm(4, 4, 6, 16, 4, 2), None),
    _diff(_att(2, 2, 20, 16, 2.5, 5, rot=_rot(80.0, 20), cap=30.0, diff=0.8), 48)])
# B: sizes that are multiples of nothing, every option that may be missing is missing, one tap, one group, one part in the norm,
# as many kept tokens as the window has, a model that starts with a parallel layer and multiplies nothing.
BB = _model(70, 157, 1e-6, 1.0, 1.0, [
    _par(_att(3, 3, 11, 7, 3.0), _ssm(3, 1, 5, 9, 1, 1), 37),
    _diff(_att(3, 1, 9, 29, 2.0, 6, diff=0.2), None),
    _par(_att(2, 1, 18, 5, 3.0, 8, 8, _rot(50.0, 2)), _ssm(5, 5, 1, 3, 2, 5), 21),
    _diff(_att(2, 2, 7, 22, 2.0, rot=_rot(40.0, 6), diff=0.0), 33)])
# C: sizes the tensor cores take: maps of 32 and 16, values of 64 and 48, windows that end inside and past a page of 64, kept tokens
# up to and over a page, heads of which sixteen or more read one key/value head, larger states.
BC = _model(128, 300, 1e-5, 0.5, 4.0, [
    _diff(_att(8, 2, 32, 64, 3.0, 70, rot=_rot(1e4, 16), cap=20.0, diff=0.5), 128),
    _par(_att(20, 1, 48, 80, 4.0, 33, 64, _rot(1e5, 32, (2.0, 128, 16.0, 2.0))), _ssm(8, 2, 40, 24, 4, 4), 160),
    _diff(_att(24, 2, 16, 48, 3.0, 90, rot=_rot(1e4, 16), cap=5.0, diff=0.7), 64),
    _par(_att(4, 4, 80, 32, 4.0, 64, 70, _rot(1e4, 80)), _ssm(4, 1, 96, 40, 2, 1), 64)])
# One mechanism alone.
B_DIFF = _model(48, 97, 1e-5, 0.9, 3.0, [_diff(_att(4, 2, 16, 16, 4.0, 25, rot=_rot(100.0, 8), cap=40.0, diff=0.3), None)])
B_PAR = _model(48, 97, 1e-5, 0.9, 3.0, [_par(_att(4, 2, 16, 16, 5.0, 25, 9, _rot(100.0, 8, (3.0, 40, 6.0, 1.0))), _ssm(4, 2, 8, 12, 3, 2), None)])
B_FF = _model(48, 97, 1e-5, 0.8, 2.0, [_diff(_att(1, 1, 4, 4, 2.0, 3, diff=0.5), 80)])
CONFIGS = {"a": BA, "b": BB, "c": BC, "diff": B_DIFF, "par": B_PAR, "ff": B_FF}


def tensor_table(config):
    """(stored name, shape) of every tensor of a model folder, from the configuration alone."""
    w = config["width"]
    out = [("embed", (config["vocab"], w)), ("final.norm", (w,))]
    for i, layer in enumerate(config["layers"]):
        m, mlp, p, x = layer["mixer"], layer.get("mlp"), f"l{i}.", f"l{i}.mix."
        out += [(p + "norm1", (w,)), (p + "ls1", (w,))]
        if layer["type"] == "attention":
            nv = m["heads"] * m["vdim"]
            out += [(x + "q", (2 * m["heads"] * m["dim"], w)), (x + "k", (2 * m["kv_heads"] * m["dim"], w)),
                    (x + "v", (m["kv_heads"] * m["vdim"], w)), (x + "g", (nv, w)), (x + "o", (w, nv))]
            out += [(x + n, (m["dim"],)) for n in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2")]
        else:
            a, r = m["left"], m["right"]
            nv, inner = a["heads"] * a["vdim"], r["heads"] * r["vdim"]
            c = inner + 2 * r["groups"] * r["state"]
            out += [(x + "left.q", (a["heads"] * a["dim"], w)), (x + "left.k", (a["kv_heads"] * a["dim"], w)),
                    (x + "left.v", (a["kv_heads"] * a["vdim"], w)), (x + "left.g", (nv, w)), (x + "left.o", (w, nv)),
                    (x + "left.out", (w,)), (x + "right.out", (w,)), (x + "right.in", (inner + c + r["heads"], w)),
                    (x + "right.conv", (c, r["conv"])), (x + "right.conv.b", (c,)), (x + "right.norm", (inner,)),
                    (x + "right.o", (w, inner))]
            out += [(x + "right." + n, (r["heads"],)) for n in ("dt_bias", "A_log", "D")]
        if mlp is not None:
            out += [(p + "norm2", (w,)), (p + "ls2", (w,)), (p + "mlp.up", (mlp["ff"], w)), (p + "mlp.down", (w, mlp["ff"]))]
    return out


def make_weights(config, seed: int):
    """Random weights, rounded to bfloat16 (so that both sides read the same numbers). Products' weights are N(0, 1/in); with the
    configurations' score scales the scores spread over several units, so a wrong key, page or window edge moves the logits. The
    embedding's rows are small beside what the layers add, so that the next token is not simply the last one again. Norm weights,
    layer scales, the two sides' weights and skips differ from one another visibly, λ is far from 0 and from `diff`, biases of the
    convolution and of the step sizes are of their inputs' size, rates spread so that some heads forget within a few tokens and
    others keep what the first tokens wrote."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_table(config):
        x = torch.randn(shape, generator=g, dtype=torch.float32)
        tail = name.split(".", 1)[1] if name.startswith("l") else name
        if name == "embed":
            x = 0.3 * x / float(config["embedding"]["scale"])
        elif tail.endswith(".conv"):
            x = 0.6 * x
        elif tail.endswith(".conv.b"):
            x = 0.5 * x
        elif tail.endswith("A_log"):
            x = -1.0 + 1.5 * x
        elif tail.endswith("dt_bias"):
            x = x - 0.5
        elif tail in ("mix.lq1", "mix.lk1", "mix.lq2", "mix.lk2"):
            x = 0.5 * x / shape[0] ** 0.25
        elif len(shape) == 1:
            x = 1.0 + 0.3 * x
        else:
            x = x / shape[1] ** 0.5
        out[name] = x.to(torch.bfloat16).contiguous()
    return out


def make_folder(tmp_path, name: str, seed: int = 0, config=None, weights=None):
    config = config or CONFIGS[name]
    folder = tmp_path / f"bukuvik_{name}"
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(config))
    save_file(weights if weights is not None else make_weights(config, seed), str(folder / "model.safetensors"))
    return folder


def read_folder(folder):
    import pathlib
    folder = pathlib.Path(folder)
    return json.loads((folder / "config.json").read_text()), load_file(str(folder / "model.safetensors"))


def exact_logits(folder, ids):
    config, weights = read_folder(folder)
    return plain.forward(weights, config, list(ids)).float()


def point_at(config, weights, ids, reads: int, key: int, size: float = 8.0):
    """The FIRST layer's attention changed so that the query at `reads` puts nearly all its weight on the key at `key` in every
    head (of two maps: in the first) if it sees it: the two tokens' rows get a large share of one channel that does not turn,
    in the query's and the key's projection. The tokens at both places must stand nowhere else. Returns new weights."""
    layer = config["layers"][0]
    m, p = (layer["mixer"], "l0.mix.") if layer["type"] == "attention" else (layer["mixer"]["left"], "l0.mix.left.")
    maps = 2 if layer["type"] == "attention" else 1
    out = {k: v.clone() for k, v in weights.items()}
    x = weights["embed"].double() * float(config["embedding"]["scale"])
    for name, heads, token in (("q", m["heads"], ids[reads]), ("k", m["kv_heads"], ids[key])):
        w = weights[p + name].double().view(heads, maps, m["dim"], -1).clone()
        w[:, 0, m["dim"] - 1] += size * x[token] / (x[token] @ x[token])
        out[p + name] = w.view(heads * maps * m["dim"], -1).to(torch.bfloat16)
    return out


# The measure, per row: the distance from the plain implementation's 64-bit logits (mean taken off, root mean square over the
# vocabulary) relative to the row's own spread. float32: every row within 2e-4. bfloat16: rounding alone leaves most rows 0.005 to
# 0.03 away; scores are sharp on purpose, so here and there a row turns on two keys a rounding apart and lands further off, in the
# plain twins of the kernels just as on the GPU. So: the median within 0.03, at most one row in fifteen beyond 0.1, none beyond 0.5.
# A wrong key, state, slot or weight moves every row it touches by a good part of its spread, and in 32-bit, where the same
# schedules run, nothing is excused.
LIMITS = {"float32": 2e-4, "bfloat16": 0.1}


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
        assert worst[0] <= 0.5, f"request {worst[1]} position {worst[2]}: error {worst[0]:.3g} of the row's spread"
        over = [e for e in errors if e[0] > LIMITS[dtype]]
        assert len(over) <= max(1, len(errors) // 15), f"{len(over)} of {len(errors)} rows are beyond {LIMITS[dtype]}: {over[-5:]}"
        assert errors[len(errors) // 2][0] <= 0.03, f"the median row is {errors[len(errors) // 2][0]:.3g} of its spread off"
        return
    assert worst[0] <= LIMITS[dtype], f"request {worst[1]} position {worst[2]}: error {worst[0]:.3g} of the row's spread"

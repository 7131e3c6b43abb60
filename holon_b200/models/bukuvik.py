"""Bukuvik: its typed configuration and its recipe.

A decoder whose config.json lists its layers one by one (`layers[i]`: `type`, the mixer's sizes under `mixer`, the feed-forward
under `mlp` or null). The embedding is scaled; norms stand on the sublayers' outputs, with a layer scale and a residual
multiplier: x ← x + m · a1 ∘ N(mixer(x)), then x ← x + m · a2 ∘ N(ff(x)), m = `residual_mult` (block `outnorm`). Mixer types:
`attention` (differential attention: two maps a head over the same values, a per-head RMS norm of q and k, a partial rotation, a
soft limit on scores, a sliding window and an output gate: mixer `maps`) and `parallel` (two mixers side by side, each under an
RMS norm of its own, half their sum: `left`, attention with YaRN's frequencies, q and k divided by their root mean square behind
the rotation, a window that keeps the sequence's first tokens and an output gate; `right`, a state space in the matrix form of
Mamba-2: mixers `maps` and `state_space`). Feed-forwards are W_down relu(W_up x)². The head is the embedding table.

Keys read: `architecture`, `width`, `vocab`, `norm.eps`, `residual_mult`, `embedding.scale`, `layers[i].{type, mixer, mlp.{kind,
ff}}`; attention: `mixer.{heads, kv_heads, dim, vdim, scale, softcap, diff, mask.size, rot.{base, dims}}`; parallel:
`mixer.left.{heads, kv_heads, dim, vdim, scale, mask.{size, keep_first}, rot.{base, dims, scaling.{factor, original, fast,
slow}}}`, `mixer.right.{heads, groups, state, vdim, conv, norm_groups}`. A missing `mask` is a layer that sees every earlier
token, a missing `keep_first` none kept, a missing `softcap` no limit, a missing `rot` no rotation, a missing `scaling` a plain
one. Stored tensors: `embed`, `final.norm`, `l<i>.{norm1, norm2, ls1, ls2}`, `l<i>.mix.{q, k, v, g, o, q.norm, k.norm, lq1, lk1,
lq2, lk2}` (attention), `l<i>.mix.left.{q, k, v, g, o, out}`, `l<i>.mix.right.{in, conv, conv.b, dt_bias, A_log, D, norm, o,
out}` (parallel), `l<i>.mlp.{up, down}`.
"""
from __future__ import annotations

import dataclasses
from collections.abc import Mapping
from typing import Any

from ..config.registry import ConfigError, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartRef, Run, WeightRule
from .rulorax import _get

PAIR_SCALE = 0.5                      # a parallel layer adds half of each side


@dataclasses.dataclass(frozen=True)
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int                          # query/key size, of one map
    vdim: int
    scale: float
    window: int                       # 0: every earlier token is seen
    keep_first: int                   # first tokens that stay visible beside the window
    rot_base: float
    rot_dims: int                     # 0: no rotation
    yarn: tuple[float, float, float, float] | None      # factor, original, fast, slow
    softcap: float | None = None
    diff: float | None = None         # given: two maps a head


@dataclasses.dataclass(frozen=True)
class StateSizes:
    heads: int
    groups: int
    state: int
    vdim: int
    taps: int
    norm_groups: int


@dataclasses.dataclass(frozen=True)
class PairSizes:
    left: AttentionSizes
    right: StateSizes


@dataclasses.dataclass(frozen=True)
class BukuvikLayer:
    kind: str                         # "attention" | "parallel"
    mixer: AttentionSizes | PairSizes
    ff: int | None


def _attention(m, where: str, two_maps: bool) -> AttentionSizes:
    mask, rot = m.get("mask"), m.get("rot")
    scaling = rot.get("scaling") if isinstance(rot, Mapping) else None
    ws = where + ".rot.scaling"
    number = lambda key: _get(m, key, float, where) if m.get(key) is not None else None      # noqa: E731
    out = AttentionSizes(
        heads=_get(m, "heads", int, where), kv_heads=_get(m, "kv_heads", int, where), dim=_get(m, "dim", int, where),
        vdim=_get(m, "vdim", int, where), scale=_get(m, "scale", float, where),
        window=_get(mask, "size", int, where + ".mask") if mask is not None else 0,
        keep_first=_get(mask, "keep_first", int, where + ".mask") if mask is not None and mask.get("keep_first") is not None else 0,
        rot_base=_get(rot, "base", float, where + ".rot") if rot is not None else 0.0,
        rot_dims=_get(rot, "dims", int, where + ".rot") if rot is not None else 0,
        yarn=tuple(_get(scaling, key, float, ws) for key in ("factor", "original", "fast", "slow")) if scaling is not None else None,
        softcap=number("softcap"), diff=_get(m, "diff", float, where) if two_maps else None)
    if min(out.heads, out.kv_heads, out.dim, out.vdim) < 1 or out.heads % out.kv_heads:
        raise ConfigError(f"config.json: {where}: sizes must be positive and heads a multiple of kv_heads")
    if not out.scale > 0 or (out.softcap is not None and not out.softcap > 0):
        raise ConfigError(f"config.json: {where}: scale and softcap must be positive")
    if mask is not None and (out.window < 1 or out.keep_first < 0):
        raise ConfigError(f"config.json: {where}.mask: size must be at least 1, keep_first not negative")
    if out.rot_dims % 2 or not 0 <= out.rot_dims <= out.dim:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim")
    if out.rot_dims and not out.rot_base > (1.0 if out.yarn else 0.0):
        raise ConfigError(f"config.json: {where}.rot.base must be positive, and above 1 with a scaling")
    if out.yarn is not None and min(out.yarn) <= 0:
        raise ConfigError(f"config.json: {ws}: every number must be positive")
    return out


def _state(m, where: str) -> StateSizes:
    out = StateSizes(heads=_get(m, "heads", int, where), groups=_get(m, "groups", int, where), state=_get(m, "state", int, where),
                     vdim=_get(m, "vdim", int, where), taps=_get(m, "conv", int, where),
                     norm_groups=_get(m, "norm_groups", int, where))
    if min(dataclasses.astuple(out)) < 1 or out.heads % out.groups or (out.heads * out.vdim) % out.norm_groups:
        raise ConfigError(f"config.json: {where}: sizes must be positive, heads a multiple of groups, and heads times vdim one of "
                          f"norm_groups")
    return out


@dataclasses.dataclass(frozen=True)
class BukuvikConfig:
    width: int
    vocab: int
    eps: float
    residual_mult: float
    embed_scale: float
    layers: tuple[BukuvikLayer, ...]
    eos_token_ids: tuple[int, ...] = ()

    @staticmethod
    def from_dict(c: Mapping[str, Any]) -> "BukuvikConfig":
        listed = c.get("layers")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError("config.json: 'layers' must list the layers")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            kind = _get(entry, "type", str, where)
            m, wm = _get(entry, "mixer", Mapping, where), where + ".mixer"
            if kind == "attention":
                mixer = _attention(m, wm, two_maps=True)
            elif kind == "parallel":
                mixer = PairSizes(_attention(_get(m, "left", Mapping, wm), wm + ".left", two_maps=False),
                                  _state(_get(m, "right", Mapping, wm), wm + ".right"))
            else:
                raise NotImplementedError(f"bukuvik: {where} has mixer type {kind!r}; known: attention, parallel")
            mlp, ff = entry.get("mlp"), None
            if mlp is not None:
                mkind = _get(mlp, "kind", str, where + ".mlp")
                if mkind != "dense":
                    raise NotImplementedError(f"bukuvik: {where}.mlp.kind {mkind!r}; known: dense")
                ff = _get(mlp, "ff", int, where + ".mlp")
                if ff < 1:
                    raise ConfigError(f"config.json: {where}.mlp.ff must be positive")
            layers.append(BukuvikLayer(kind, mixer, ff))
        eos = c.get("eos_token_id", ())
        eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
        cfg = BukuvikConfig(width=_get(c, "width", int, "config"), vocab=_get(c, "vocab", int, "config"),
                            eps=_get(_get(c, "norm", Mapping, "config"), "eps", float, "norm"),
                            residual_mult=_get(c, "residual_mult", float, "config"),
                            embed_scale=_get(_get(c, "embedding", Mapping, "config"), "scale", float, "embedding"),
                            layers=tuple(layers), eos_token_ids=eos)
        if cfg.width < 1 or cfg.vocab < 1:
            raise ConfigError("config.json: 'width' and 'vocab' must be positive")
        return cfg


WEIGHT_RULES = (
    WeightRule("embed", "embed.weight"),
    WeightRule("final.norm", "norm.weight"),
    WeightRule("l{i}.norm1", "layers.{i}.mixer_norm.weight"),
    WeightRule("l{i}.norm2", "layers.{i}.ffn_norm.weight"),
    WeightRule("l{i}.ls1", "layers.{i}.mixer_scale"),
    WeightRule("l{i}.ls2", "layers.{i}.ffn_scale"),
    WeightRule("l{i}.mix.{rest}", "layers.{i}.mixer.{rest}"),
    WeightRule("l{i}.mlp.{rest}", "layers.{i}.ffn.{rest}"),
)


def _maps_ref(cfg: BukuvikConfig, m: AttentionSizes) -> PartRef:
    position = PartRef.of("position", "rope", theta=m.rot_base, rotary_dim=m.rot_dims, yarn=m.yarn) if m.rot_dims else None
    return PartRef.of("mixer", "maps", heads=m.heads, kv_heads=m.kv_heads, key_dim=m.dim, value_dim=m.vdim, scale=m.scale,
                      eps=cfg.eps, maps=1 if m.diff is None else 2, diff=m.diff, softcap=m.softcap, window=m.window,
                      keep_first=m.keep_first, qk_norm="after" if m.diff is None else "before", gate=True, position=position)


def recipe(cfg: BukuvikConfig) -> ModelSpec:
    norm = PartRef.of("norm", "rmsnorm", eps=cfg.eps)
    block = PartRef.of("block", "outnorm", residual_mult=cfg.residual_mult, layer_scale=True)
    layers = []
    for layer in cfg.layers:
        if layer.kind == "attention":
            mixer = _maps_ref(cfg, layer.mixer)
        else:
            r = layer.mixer.right
            right = PartRef.of("mixer", "state_space", heads=r.heads, vdim=r.vdim, state=r.state, groups=r.groups, taps=r.taps,
                               norm_groups=r.norm_groups, eps=cfg.eps)
            mixer = PartRef.of("mixer", "side_by_side", left=_maps_ref(cfg, layer.mixer.left), right=right, left_scale=PAIR_SCALE,
                               right_scale=PAIR_SCALE, out_eps=cfg.eps)
        ffn = PartRef.of("ffn", "mlp", inter=layer.ff, activation="relu2") if layer.ff is not None else None
        layers.append(LayerSpec(block, mixer, ffn, norm))
    return ModelSpec(hidden=cfg.width, vocab=cfg.vocab, layers=tuple(layers), order=tuple(Run(i, i) for i in range(len(layers))),
                     embed=PartRef.of("embed", "pair", scale=cfg.embed_scale), norm=norm,
                     head=PartRef.of("head", "linear", tied=True), weight_rules=WEIGHT_RULES)


register_architecture("Bukuvik", BukuvikConfig.from_dict, recipe)

"""Gegunex: its typed configuration and its recipe.

A decoder whose config.json lists its layers one by one (`layers[i]`: `type`, the mixer's sizes under `mixer`, the
feed-forward under `mlp` or null). Blocks are pre-norm with a factor on what is added: x ← x + m · mixer(N1(x)), then
x ← x + m · ff(N2(x)), m = `residual_mult`, N a layer norm with a weight and no bias. Mixer types: `lightning` (linear attention
over a matrix state per head with one fixed decay a head; q, k, v pass silu; one norm over all heads and a sigmoid gate),
`latent_attention` (queries and keys/values each through a normed latent, a rotated part of neighbouring pairs with YaRN's
frequencies, a sliding window, a sink in the softmax; only the latent and the shared rotated key part are cached) and
`channel_delta` (a gated delta rule with a decay per key channel behind short convolutions). Feed-forwards are routed experts:
clamped gated units, sigmoid scores, the `top` largest, each score multiplying its expert's input. The head is the
embedding table, and the logits pass a soft limit.

Keys read: `architecture`, `width`, `vocab`, `norm.eps`, `residual_mult`, `logit_softcap`, `layers[i].{type, mixer, mlp}`;
lightning: `mixer.{heads, dim, vdim, decay}`; latent_attention: `mixer.{heads, dim, rot_dim, vdim, q_rank, kv_rank, scale,
mask.size, rot.{base, dims, scaling.{factor, original, fast, slow}}}`; channel_delta: `mixer.{heads, kv_heads, dim, vdim,
conv}`; `mlp.{kind, expert.{ff, limit}, router.{experts, top}}`. A missing `scaling` is a plain rotation, a missing `mask` a layer
that sees every earlier token. Two sizes stand in no key of a stored model's config.json, the ranks of the delta rule's
low-rank decay and gate projections: `complete` reads them from the shapes of `l<i>.mix.a1` and `.g1` and enters them as
`mixer.decay_rank` and `mixer.gate_rank` (a config dict made by hand, for random weights, gives them itself).
Stored tensors: `embed`, `final.norm`, `l<i>.{norm1, norm2}`, `l<i>.mix.{q, k, v, g, norm, o}` (lightning), `l<i>.mix.{dq,
dq.norm, uq, dkv, dkv.norm, uk, uv, sink, o}` (latent_attention), `l<i>.mix.{q, k, v, q.conv, k.conv, v.conv, b, a1, a2, dt_bias,
A_log, g1, g2, norm, o}` (channel_delta), `l<i>.mlp.{router, e<j>.{gate, up, down}}`.
"""
from __future__ import annotations

import copy
import dataclasses
from collections.abc import Mapping
from typing import Any

from ..config.registry import ConfigError, register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartRef, Run, WeightRule
from .rulorax import _get

GATE_SLOPE = 1.702                    # a clamped unit's gate is g · sigmoid(GATE_SLOPE · g)


@dataclasses.dataclass(frozen=True)
class LightningSizes:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]


@dataclasses.dataclass(frozen=True)
class LatentSizes:
    heads: int
    dim: int                      # unrotated query/key dimensions per head
    rot_dim: int                  # rotated ones (the key's are shared by all heads)
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int                   # 0: every earlier token is seen
    rot_base: float
    rot_dims: int
    yarn: tuple[float, float, float, float] | None      # factor, original, fast, slow


@dataclasses.dataclass(frozen=True)
class DeltaSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int
    gate_rank: int


@dataclasses.dataclass(frozen=True)
class ExpertUnits:
    experts: int
    top: int
    ff: int
    limit: float


@dataclasses.dataclass(frozen=True)
class GegunexLayer:
    kind: str                     # "lightning" | "latent_attention" | "channel_delta"
    mixer: LightningSizes | LatentSizes | DeltaSizes
    mlp: ExpertUnits | None


def _lightning(m, where: str) -> LightningSizes:
    decay = _get(m, "decay", (list, tuple), where)
    if not all(isinstance(d, (int, float)) and not isinstance(d, bool) for d in decay):
        raise ConfigError(f"config.json: {where}.decay must list numbers")
    out = LightningSizes(heads=_get(m, "heads", int, where), dim=_get(m, "dim", int, where), vdim=_get(m, "vdim", int, where),
                         decay=tuple(float(d) for d in decay))
    if min(out.heads, out.dim, out.vdim) < 1 or len(out.decay) != out.heads:
        raise ConfigError(f"config.json: {where}: sizes must be positive and decay list one number per head")
    return out


def _latent(m, where: str) -> LatentSizes:
    rot, mask = m.get("rot"), m.get("mask")
    scaling = rot.get("scaling") if isinstance(rot, Mapping) else None
    ws = where + ".rot.scaling"
    out = LatentSizes(
        heads=_get(m, "heads", int, where), dim=_get(m, "dim", int, where), rot_dim=_get(m, "rot_dim", int, where),
        vdim=_get(m, "vdim", int, where), q_rank=_get(m, "q_rank", int, where), kv_rank=_get(m, "kv_rank", int, where),
        scale=_get(m, "scale", float, where), window=_get(mask, "size", int, where + ".mask") if mask is not None else 0,
        rot_base=_get(rot, "base", float, where + ".rot") if rot is not None else 0.0,
        rot_dims=_get(rot, "dims", int, where + ".rot") if rot is not None else 0,
        yarn=tuple(_get(scaling, key, float, ws) for key in ("factor", "original", "fast", "slow")) if scaling is not None else None)
    if min(out.heads, out.dim, out.vdim, out.q_rank, out.kv_rank) < 1 or out.rot_dim < 0:
        raise ConfigError(f"config.json: {where}: every size must be positive")
    if mask is not None and out.window < 1:
        raise ConfigError(f"config.json: {where}.mask.size must be at least 1")
    if out.rot_dims % 2 or not 0 <= out.rot_dims <= out.rot_dim:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most rot_dim")
    if out.rot_dims and not out.rot_base > (1.0 if out.yarn else 0.0):
        raise ConfigError(f"config.json: {where}.rot.base must be positive, and above 1 with a scaling")
    if out.yarn is not None and min(out.yarn) <= 0:
        raise ConfigError(f"config.json: {ws}: every number must be positive")
    return out


def _delta(m, where: str) -> DeltaSizes:
    for name, stored in (("decay_rank", "a1"), ("gate_rank", "g1")):
        if name not in m:
            raise ConfigError(f"config.json: {where}.{name} is given neither by the dict nor by a stored tensor's shape "
                              f"(l<i>.mix.{stored})")
    out = DeltaSizes(heads=_get(m, "heads", int, where), kv_heads=_get(m, "kv_heads", int, where), dim=_get(m, "dim", int, where),
                     vdim=_get(m, "vdim", int, where), taps=_get(m, "conv", int, where),
                     decay_rank=_get(m, "decay_rank", int, where), gate_rank=_get(m, "gate_rank", int, where))
    if min(dataclasses.astuple(out)) < 1 or out.heads % out.kv_heads:
        raise ConfigError(f"config.json: {where}: sizes must be positive and heads a multiple of kv_heads")
    return out


_MIXERS = {"lightning": _lightning, "latent_attention": _latent, "channel_delta": _delta}


@dataclasses.dataclass(frozen=True)
class GegunexConfig:
    width: int
    vocab: int
    eps: float
    residual_mult: float
    softcap: float
    layers: tuple[GegunexLayer, ...]
    eos_token_ids: tuple[int, ...] = ()

    @staticmethod
    def from_dict(c: Mapping[str, Any]) -> "GegunexConfig":
        listed = c.get("layers")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError("config.json: 'layers' must list the layers")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            kind = _get(entry, "type", str, where)
            if kind not in _MIXERS:
                raise NotImplementedError(f"gegunex: {where} has mixer type {kind!r}; known: {', '.join(sorted(_MIXERS))}")
            mixer = _MIXERS[kind](_get(entry, "mixer", Mapping, where), where + ".mixer")
            mlp, unit = entry.get("mlp"), None
            if mlp is not None:
                wf = where + ".mlp"
                mkind = _get(mlp, "kind", str, wf)
                if mkind != "moe":
                    raise NotImplementedError(f"gegunex: {wf}.kind {mkind!r}; known: moe")
                router, expert = _get(mlp, "router", Mapping, wf), _get(mlp, "expert", Mapping, wf)
                unit = ExpertUnits(experts=_get(router, "experts", int, wf + ".router"), top=_get(router, "top", int, wf + ".router"),
                                   ff=_get(expert, "ff", int, wf + ".expert"), limit=_get(expert, "limit", float, wf + ".expert"))
                if unit.ff < 1 or not 1 <= unit.top <= unit.experts or not unit.limit > 0:
                    raise ConfigError(f"config.json: {wf}: ff and limit must be positive and 1 <= top <= experts")
            layers.append(GegunexLayer(kind, mixer, unit))
        eos = c.get("eos_token_id", ())
        eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
        cfg = GegunexConfig(width=_get(c, "width", int, "config"), vocab=_get(c, "vocab", int, "config"),
                            eps=_get(_get(c, "norm", Mapping, "config"), "eps", float, "norm"),
                            residual_mult=_get(c, "residual_mult", float, "config"),
                            softcap=_get(c, "logit_softcap", float, "config"), layers=tuple(layers), eos_token_ids=eos)
        if cfg.width < 1 or cfg.vocab < 1 or not cfg.softcap > 0:
            raise ConfigError("config.json: 'width', 'vocab' and 'logit_softcap' must be positive")
        return cfg


def complete(c: Mapping[str, Any], shapes: Mapping[str, tuple]) -> dict[str, Any]:
    """config.json with the delta-rule layers' `decay_rank` and `gate_rank` entered from the stored tensors' shapes."""
    c = copy.deepcopy(dict(c))
    listed = c.get("layers")
    for i, entry in enumerate(listed if isinstance(listed, list) else ()):
        if not isinstance(entry, dict) or entry.get("type") != "channel_delta" or not isinstance(entry.get("mixer"), dict):
            continue
        for key, stored in (("decay_rank", f"l{i}.mix.a1"), ("gate_rank", f"l{i}.mix.g1")):
            if key not in entry["mixer"] and stored in shapes:
                entry["mixer"][key] = int(shapes[stored][0])
    return c


WEIGHT_RULES = (
    WeightRule("embed", "embed.weight"),
    WeightRule("final.norm", "norm.weight"),
    WeightRule("l{i}.norm1", "layers.{i}.input_norm.weight"),
    WeightRule("l{i}.norm2", "layers.{i}.post_norm.weight"),
    WeightRule("l{i}.mix.{rest}", "layers.{i}.mixer.{rest}"),
    WeightRule("l{i}.mlp.{rest}", "layers.{i}.ffn.{rest}"),
)


def _mixer_ref(cfg: GegunexConfig, layer: GegunexLayer) -> PartRef:
    m = layer.mixer
    if layer.kind == "lightning":
        return PartRef.of("mixer", "lightning", heads=m.heads, dim=m.dim, vdim=m.vdim, decay=m.decay, eps=cfg.eps)
    if layer.kind == "channel_delta":
        return PartRef.of("mixer", "gated_delta", heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, taps=m.taps,
                          decay_rank=m.decay_rank, gate_rank=m.gate_rank, eps=cfg.eps)
    position = PartRef.of("position", "rope", theta=m.rot_base, rotary_dim=m.rot_dims, interleaved=True, yarn=m.yarn) \
        if m.rot_dims else None
    return PartRef.of("mixer", "latent", heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, rank=m.kv_rank,
                      q_rank=m.q_rank, scale=m.scale, window=m.window, gate=False, sink=True,
                      norm=PartRef.of("norm", "rmsnorm", eps=cfg.eps), position=position)


def recipe(cfg: GegunexConfig) -> ModelSpec:
    norm = PartRef.of("norm", "layernorm", eps=cfg.eps)
    block = PartRef.of("block", "prenorm", residual_mult=cfg.residual_mult)
    layers = []
    for layer in cfg.layers:
        u = layer.mlp
        ffn = PartRef.of("ffn", "experts", experts=u.experts, top=u.top, scale=1.0, inter=u.ff, activation="clamped", gated=True,
                         limit=u.limit, alpha=GATE_SLOPE, scores="sigmoid", weight_on="input") if u is not None else None
        layers.append(LayerSpec(block, _mixer_ref(cfg, layer), ffn, norm))
    return ModelSpec(hidden=cfg.width, vocab=cfg.vocab, layers=tuple(layers), order=tuple(Run(i, i) for i in range(len(layers))),
                     embed=PartRef.of("embed", "table"), norm=norm,
                     head=PartRef.of("head", "linear", tied=True, softcap=cfg.softcap), weight_rules=WEIGHT_RULES)


register_architecture("Gegunex", GegunexConfig.from_dict, recipe, complete=complete)

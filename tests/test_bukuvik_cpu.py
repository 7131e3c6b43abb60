"""Bukuvik without a GPU: configuration, weight names, each mechanism alone against the written-out rule, the cache manager's kept
first pages, and the engine's host side (batch layout, cache entries with windows and kept pages, the per-request state of the
state-space layers) with the CPU twins of the kernels (tests/ref_kernels.py) against the plain implementation
(tests/plain_bukuvik.py)."""
from __future__ import annotations

import copy
import json

import numpy as np
import pytest
import torch

import plain_bukuvik as plain
from bukuvik_tools import CONFIGS, compare, exact_logits, make_folder, make_weights, point_at, read_folder, tensor_table
from helpers import random_prompt
from holon_b200.config.registry import ConfigError, resolve_architecture
from holon_b200.replay import Replayer
from ref_kernels import RefKernels
from replay_tools import portions, run


def test_architecture_and_configuration():
    arch = resolve_architecture(CONFIGS["a"])
    cfg = arch.parse(CONFIGS["a"])
    assert arch.name == "Bukuvik" and len(cfg.layers) == 4 and cfg.layers[2].ff is None
    spec = arch.recipe(cfg)
    assert [(r.layer, r.cache, r.fills) for r in spec.order] == [(i, i, True) for i in range(4)]
    assert all(layer.block.name == "outnorm" and layer.norm.name == "rmsnorm" for layer in spec.layers)
    assert spec.layers[0].block.kwargs() == {"residual_mult": 0.7, "layer_scale": True}
    assert spec.head.kwargs() == {"tied": True} and spec.embed.kwargs() == {"scale": 2.5}
    assert [layer.mixer.name for layer in spec.layers] == ["maps", "side_by_side", "side_by_side", "maps"]
    m = spec.layers[0].mixer.kwargs()
    assert (m["maps"], m["diff"], m["softcap"], m["window"], m["keep_first"], m["qk_norm"]) == (2, 0.4, 6.0, 10, 0, "before")
    side = spec.layers[1].mixer.kwargs()
    left, right = side["left"].kwargs(), side["right"].kwargs()
    assert side["left_scale"] == side["right_scale"] == 0.5 and side["out_eps"] == 1e-5
    assert (left["maps"], left["diff"], left["softcap"], left["window"], left["keep_first"], left["qk_norm"]) == (1, None, None, 7, 6, "after")
    assert left["position"].kwargs()["yarn"] == (4.0, 64.0, 8.0, 1.0) and left["position"].kwargs()["rotary_dim"] == 12
    assert (right["heads"], right["groups"], right["state"], right["vdim"], right["taps"], right["norm_groups"]) == (6, 2, 10, 8, 3, 3)
    assert spec.layers[1].ffn.kwargs() == {"inter": 72, "activation": "relu2"}
    for path, value, error in (
            (("layers", 0, "type"), "retention", NotImplementedError),
            (("layers", 0, "mlp", "kind"), "moe", NotImplementedError),
            (("layers", 0, "mlp", "ff"), 0, ConfigError),
            (("layers", 0, "mixer", "kv_heads"), 3, ConfigError),
            (("layers", 0, "mixer", "diff"), None, ConfigError),
            (("layers", 0, "mixer", "softcap"), 0.0, ConfigError),
            (("layers", 0, "mixer", "scale"), -1.0, ConfigError),
            (("layers", 0, "mixer", "mask", "size"), 0, ConfigError),
            (("layers", 0, "mixer", "rot", "dims"), 14, ConfigError),
            (("layers", 0, "mixer", "rot", "dims"), 5, ConfigError),
            (("layers", 1, "mixer", "left", "mask", "keep_first"), -1, ConfigError),
            (("layers", 1, "mixer", "left", "rot", "scaling", "factor"), 0.0, ConfigError),
            (("layers", 1, "mixer", "left", "rot", "scaling"), {"factor": 2.0}, ConfigError),
            (("layers", 1, "mixer", "right", "groups"), 4, ConfigError),
            (("layers", 1, "mixer", "right", "norm_groups"), 5, ConfigError),
            (("layers", 1, "mixer", "right", "conv"), 0, ConfigError),
            (("layers", 1, "mixer", "right"), None, ConfigError),
            (("residual_mult",), None, ConfigError),
            (("width",), 0, ConfigError)):
        c = copy.deepcopy(CONFIGS["a"])
        at = c
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(error):
            arch.parse(c)
    b = arch.parse(CONFIGS["b"])                            # what may be missing is: no mask, cap, rotation, scaling, kept tokens
    assert (b.layers[0].mixer.left.window, b.layers[0].mixer.left.rot_dims, b.layers[1].mixer.softcap, b.layers[1].mixer.keep_first) == (0, 0, None, 0)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_and_shapes(name):
    from holon_b200.weights import RandomSource
    table = {stored: tuple(shape) for stored, shape, _ in RandomSource(CONFIGS[name], 0).table()}
    assert table == dict(tensor_table(CONFIGS[name]))


def test_a_missing_a_misshapen_and_a_spare_tensor_are_named(tmp_path):
    from safetensors.torch import load_file, save_file
    from holon_b200.weights.loader import WeightError
    folder = make_folder(tmp_path, "a")
    tensors = load_file(str(folder / "model.safetensors"))
    del tensors["l1.mix.right.out"]
    tensors["l0.mix.q.norm"] = torch.zeros(3, dtype=torch.bfloat16)
    tensors["l2.ls2"] = tensors["l0.ls2"].clone()                         # layer 2 has no feed-forward
    save_file(tensors, str(folder / "model.safetensors"))
    with pytest.raises(WeightError) as e:
        Replayer(str(folder), "float32", 64, device="cpu", kernels=RefKernels())
    assert e.value.missing == ["l1.mix.right.out"] and e.value.unexpected == ["l2.ls2"]
    assert [s[0] for s in e.value.shapes] == ["l0.mix.q.norm"]


# ---------------------------------------------------------------- kept first pages
def test_kept_first_pages_stay_and_the_gap_behind_them_is_given_back():
    from holon_b200.cache import CacheManager
    from holon_b200.parts.base import PagedRows
    from holon_b200.parts.model import CacheEntry
    entries = [CacheEntry(0, 0, PagedRows(1, 4, 4, window=6, keep_first=5), ()), CacheEntry(1, 1, PagedRows(1, 4, 4, window=6), ())]
    c = CacheManager(entries, 4, 2, 64, torch.float32, "cpu", pages=16)
    kept, plain_group = c.groups
    assert kept.kept == 2 and plain_group.kept == 0
    a, b = c.admit(), c.admit()
    for tokens in range(1, 41):
        assert c.reserve(a, tokens)
        c.advance(a, tokens)
        c.check()
        lo = max(0, tokens - 6 + 1) // 4                                  # the first page the next token's window reaches
        held = [i for i in range(10) if kept.table[a, i] != kept.null_page]
        assert held == sorted(set(range(min(2, kept.count[a]))) | set(range(lo, int(kept.count[a]))))
        assert [i for i in range(10) if plain_group.table[a, i] != plain_group.null_page] == list(range(lo, int(kept.count[a])))
    assert c.reserve(b, 48) and not c.reserve(a, 56)                      # b's 12 pages and a's 4 fill the pool
    assert c.could_fit(b, 60, releasing=[a])
    c.check()
    c.release(a)
    c.check()
    assert c.reserve(b, 60) and kept.pool.available == 1
    c.release(b)
    c.check()
    assert kept.pool.available == plain_group.pool.available == 16
    one = PagedRows(1, 4, 4, window=0, keep_first=5)                      # without a window nothing is passed, and nothing kept apart
    assert CacheManager([CacheEntry(0, 0, one, ())], 4, 2, 64, torch.float32, "cpu", pages=16).groups[0].kept == 0


def test_prefix_pages_of_a_group_with_kept_first_positions():
    """The index asks such a group for every page of a prefix, as one without a window; a request that has passed pages enters
    only what it holds."""
    from holon_b200.cache import CacheManager
    from holon_b200.parts.base import PagedRows
    from holon_b200.parts.model import CacheEntry
    c = CacheManager([CacheEntry(0, 0, PagedRows(1, 4, 4, window=6, keep_first=5), ())], 4, 3, 64, torch.float32, "cpu", pages=20,
                     prefix_cache=True)
    tokens = list(range(30))
    a = c.admit(tokens)
    assert c.reserve(a, 12)
    c.advance(a, 12)
    c.publish(a, tokens)
    c.check()
    b = c.admit(tokens)
    assert int(c.computed[b]) == 12 and [int(x) for x in c.groups[0].table[b, :3]] == [int(x) for x in c.groups[0].table[a, :3]]
    for slot in (a, b):
        assert c.reserve(slot, 30)
        c.advance(slot, 30)
        c.check()
    c.release(a)
    c.release(b)
    c.check()


# ---------------------------------------------------------------- mechanisms alone
def _rows(counts, held, slots, table):
    import types
    qs = np.concatenate(([0], np.cumsum(counts)))
    t = lambda x: torch.tensor(np.asarray(x), dtype=torch.int32)          # noqa: E731
    return types.SimpleNamespace(query_start=t(qs), row_slot=t(slots), kv_len=t(held), n_rows=len(counts), n_tokens=int(qs[-1]),
                                 n_decode=sum(1 for n in counts if n == 1))


def _load(part, g, scale=1.0):
    weights = {}
    for name, p, (r0, r1) in part.loadables():
        if p.tensor is None:
            p.tensor = torch.empty(p.shape)
        shape = p.piece_shape((r0, r1))
        weights[name] = torch.randn(shape, generator=g) * (scale / shape[-1] ** 0.5 if len(shape) > 1 else 0.4) + (0.0 if len(shape) > 1 or name[:2] in ("lq", "lk") else 0.7)
        p.tensor[r0:r1] = weights[name]
    part.finalize()
    return weights


def test_two_maps_are_subtracted_normed_scaled_and_gated():
    """One attention mixer over a whole sequence against the written-out rule, and that it is none of its near misses."""
    from holon_b200.config.spec import PartRef
    from holon_b200.parts.base import BuildContext
    from holon_b200.parts.model import LayerCache
    import types
    m = CONFIGS["diff"]["layers"][0]["mixer"]
    ctx = BuildContext("cpu", torch.float32, RefKernels(), max_positions=64)
    rope = PartRef.of("position", "rope", theta=m["rot"]["base"], rotary_dim=m["rot"]["dims"])
    part = ctx.part(PartRef.of("mixer", "maps", heads=4, kv_heads=2, key_dim=16, value_dim=16, scale=m["scale"], eps=1e-5, maps=2,
                               diff=m["diff"], softcap=m["softcap"], window=25, qk_norm="before", position=rope), hidden=48)
    weights = _load(part, torch.Generator().manual_seed(5))
    x = torch.randn(40, 48, generator=torch.Generator().manual_seed(6))
    rows = _rows([40], [40], [0], None)
    kv = torch.zeros(11, 2, 4, 48)
    table = torch.arange(10, dtype=torch.int32)[None]
    group = types.SimpleNamespace(block_table=table, write_index=torch.arange(40, dtype=torch.int32))
    step = types.SimpleNamespace(rows=rows, positions=torch.arange(40, dtype=torch.int32))
    got = part.forward(x, step, LayerCache(kv, group, True, {})).double()
    want = plain.two_map_attention(x.double(), weights, "", m, 1e-5)
    assert torch.allclose(got, want, atol=2e-5)
    lam = float((weights["lq1"] * weights["lk1"]).sum().exp() - (weights["lq2"] * weights["lk2"]).sum().exp()) + m["diff"]
    assert abs(part.lam - lam) < 1e-5 and abs(lam - m["diff"]) > 0.05
    for change in ({"softcap": None}, {"diff": 0.6}, {"mask": {"size": 24}}, {"mask": {"size": 26}}, {"scale": m["scale"] * 1.1},
                   {"rot": {"base": 100.0, "dims": 6}}):
        assert float((plain.two_map_attention(x.double(), weights, "", {**m, **change}, 1e-5) - want).abs().max()) > 1e-3, change


def test_kept_first_tokens_and_yarn():
    m = CONFIGS["par"]["layers"][0]["mixer"]["left"]
    g = torch.Generator().manual_seed(8)
    weights = {n: torch.randn(s, 48, generator=g) / 7 for n, s in (("q", 64), ("k", 32), ("v", 32), ("g", 64))}
    weights["o"] = torch.randn(48, 64, generator=g) / 8
    x = torch.randn(60, 48, generator=g).double()
    want = plain.kept_window_attention(x, weights, "", m, 1e-5)
    for change in ({"mask": {"size": 25, "keep_first": 8}}, {"mask": {"size": 25, "keep_first": 10}}, {"mask": {"size": 25}},
                   {"mask": {"size": 24, "keep_first": 9}}, {"rot": {"base": 100.0, "dims": 8}}):
        assert float((plain.kept_window_attention(x, weights, "", {**m, **change}, 1e-5) - want)[34:].abs().max()) > 1e-3, change
    assert plain.visible(40, 8, m["mask"]) and not plain.visible(40, 9, m["mask"]) and not plain.visible(40, 15, m["mask"]) \
        and plain.visible(40, 16, m["mask"]) and not plain.visible(7, 8, m["mask"])


@pytest.mark.parametrize("heads,groups,n,vdim,taps,norm_groups", [(4, 2, 6, 5, 3, 2), (3, 1, 7, 4, 1, 1), (6, 3, 1, 2, 4, 4), (2, 2, 9, 8, 2, 1)])
def test_state_space_in_portions_against_the_written_out_rule(heads, groups, n, vdim, taps, norm_groups):
    from holon_b200.config.spec import PartRef
    from holon_b200.parts.base import BuildContext
    from holon_b200.parts.model import LayerCache
    import types
    ctx = BuildContext("cpu", torch.float32, RefKernels(), max_positions=64)
    m = dict(heads=heads, groups=groups, state=n, vdim=vdim, conv=taps, norm_groups=norm_groups)
    part = ctx.part(PartRef.of("mixer", "state_space", heads=heads, groups=groups, state=n, vdim=vdim, taps=taps, norm_groups=norm_groups,
                               eps=1e-5), hidden=20)
    weights = _load(part, torch.Generator().manual_seed(3), scale=1.5)
    x = torch.randn(23, 20, generator=torch.Generator().manual_seed(4))
    want = plain.state_space(x.double(), weights, "", m, 1e-5)
    for cut in ([23], [1] * 23, [5, 1, 2, 2, 1, 9, 3], [2, 21]):
        slots = {s.name: torch.zeros((3, *s.shape)) for s in part.slot_states()}
        at = 0
        for size in cut:
            step = types.SimpleNamespace(rows=_rows([size], [at + size], [1], None))
            got = part.forward(x[at:at + size], step, LayerCache(None, None, True, slots)).double()
            assert torch.allclose(got, want[at:at + size], atol=2e-5), (cut, at)
            at += size
        assert all(float(t[0].abs().max()) == 0 and float(t[2].abs().max()) == 0 for t in slots.values())


def test_a_pair_of_outputs_under_other_blocks(tmp_path):
    """The two sides put together by the block's kernel, and by the mixer itself for a block that does not know the pair."""
    from holon_b200.parts.base import NormedPair
    g = torch.Generator().manual_seed(2)
    a, b, src = (torch.randn(5, 24, generator=g) for _ in range(3))
    wa, wb, w = (1 + 0.3 * torch.randn(24, generator=g) for _ in range(3))
    pair = NormedPair(a, wa, b, wb, 1e-5, 0.5)
    z = 0.5 * (plain.unit_rms(a.double(), 1e-5) * wa + plain.unit_rms(b.double(), 1e-5) * wb)
    assert torch.allclose(pair.combined().double(), z, atol=1e-6)
    dst = src.clone()
    RefKernels().out_norm_pair_add(dst, dst, pair, w, 1e-5, 0.0)
    assert torch.allclose(dst.double(), src + plain.unit_rms(z, 1e-5) * w, atol=1e-5)


# ---------------------------------------------------------------- the model through the replayer
@pytest.fixture(scope="module", params=sorted(CONFIGS))
def model(request, tmp_path_factory):
    folder = make_folder(tmp_path_factory.mktemp("models"), request.param, seed=7)
    config = CONFIGS[request.param]
    prompts = {f"r{i}": random_prompt(config["vocab"], n, 60 + i) for i, n in enumerate((23, 41, 9, 30))}
    return folder, config, prompts, {rid: exact_logits(folder, ids) for rid, ids in prompts.items()}


def test_cache_entries_and_states(model):
    folder, config, _, _ = model
    r = Replayer(str(folder), "float32", 64, device="cpu", kernels=RefKernels(), page_size=4)
    states = r.built.cache.slot_states
    assert sorted(e for g in r.built.cache.groups for e in g.entries) == list(range(len(config["layers"])))
    for i, layer in enumerate(config["layers"]):
        two = layer["type"] == "attention"
        m = layer["mixer"] if two else layer["mixer"]["left"]
        group = r.built.cache.group_of_entry[i]
        assert tuple(group.kv.shape[2:]) == (m["kv_heads"], 4, (1 + two) * m["dim"] + m["vdim"])
        mask = m.get("mask", {})
        assert group.decl.window == mask.get("size", 0) and group.kept == -(-mask.get("keep_first", 0) // 4)
        if two:
            assert not [key for key in states if key[0] == i]
            continue
        s = layer["mixer"]["right"]
        assert tuple(states[(i, "right.state")].shape[1:]) == (s["heads"], s["vdim"], s["state"]) and states[(i, "right.state")].dtype == torch.float32
        if s["conv"] > 1:
            assert tuple(states[(i, "right.conv")].shape[1:]) == (s["conv"] - 1, s["heads"] * s["vdim"] + 2 * s["groups"] * s["state"])
        else:
            assert (i, "right.conv") not in states


def test_whole_tail_portions_and_mixed(model):
    folder, config, prompts, want = model
    r = Replayer(str(folder), "float32", 64, device="cpu", kernels=RefKernels(), page_size=4)
    compare(run(r, [([(rid, ids)], [rid]) for rid, ids in prompts.items()]), want, "float32")
    steps = []
    for rid, ids in prompts.items():                                       # from the first token on, one by one
        steps += [([(rid, [t])], [rid] if i == len(ids) - 1 else []) for i, t in enumerate(ids)]
    compare(run(r, steps), want, "float32")
    steps = []
    for rid, ids in prompts.items():                                       # portions down to two tokens
        parts = portions(ids, [3, 2, 7, 2, 5])
        steps += [([(rid, p)], [rid] if i == len(parts) - 1 else []) for i, p in enumerate(parts)]
    compare(run(r, steps), want, "float32")
    # up to three requests at once in 104 tokens of pool: portions beside single tokens, pages and slots given back and used
    # again (a slot's state, its carried inputs and its pages must not leak into the request that takes it next)
    r = Replayer(str(folder), "float32", 104, device="cpu", kernels=RefKernels(), page_size=4)
    at, steps, sizes = {rid: 0 for rid in prompts}, [], {"r0": [1, 1, 4], "r1": [6, 2, 1], "r2": [2], "r3": [1, 9]}
    live, waiting, turn = ["r0", "r1", "r2"], ["r3"], 0
    while live:
        entries, end = [], []
        for rid in list(live):
            n = min(sizes[rid][turn % len(sizes[rid])], len(prompts[rid]) - at[rid])
            entries.append((rid, prompts[rid][at[rid]:at[rid] + n]))
            at[rid] += n
            if at[rid] == len(prompts[rid]):
                end.append(rid)
                live.remove(rid)
                if waiting:
                    live.append(waiting.pop())
        steps.append((entries, end))
        turn += 1
    got = run(r, steps)
    compare(got, want, "float32")
    assert len(got) == sum(len(ids) for ids in prompts.values())
    again = {"r0": prompts["r1"], "r1": prompts["r0"]}                     # the same slots and pages, other requests
    compare(run(r, [([("r0", again["r0"][:20]), ("r1", again["r1"][:3])], []),
                    ([("r0", again["r0"][20:]), ("r1", again["r1"][3:])], ["r0", "r1"])]),
            {"r0": want["r1"], "r1": want["r0"]}, "float32")


def test_a_request_alone_and_beside_others_agree(model):
    folder, config, prompts, _ = model
    alone = run(Replayer(str(folder), "float32", 64, device="cpu", kernels=RefKernels(), page_size=4),
                [([("r1", prompts["r1"])], ["r1"])])
    r = Replayer(str(folder), "float32", 128, device="cpu", kernels=RefKernels(), page_size=4)
    both = run(r, [([("r0", prompts["r0"][:7]), ("r1", prompts["r1"][:30])], []),
                   ([("r1", prompts["r1"][30:]), ("r0", prompts["r0"][7:8]), ("r2", prompts["r2"])], ["r0", "r1", "r2"])])
    for pos in range(len(prompts["r1"])):
        assert torch.allclose(alone[("r1", pos)], both[("r1", pos)], atol=2e-5 * float(alone[("r1", pos)].std()) + 2e-5, rtol=0)


def edge_cases(kind, window, keep, reads):
    """(name, the key's position, the change of the mask that must show) just inside and just outside every edge of a mask."""
    cases = [("window in", reads - window + 1, {"size": window - 1}), ("window out", reads - window, {"size": window + 1})]
    if kind == "par":
        cases += [("first in", keep - 1, {"keep_first": keep - 1}), ("first out", keep, {"keep_first": keep + 1})]
    return [c for c in cases if c[1] != reads]


def pointed(kind, window, keep, reads, key, length):
    config = copy.deepcopy(CONFIGS[kind])
    m = config["layers"][0]["mixer"] if kind == "diff" else config["layers"][0]["mixer"]["left"]
    m["mask"] = {"size": window} if kind == "diff" else {"size": window, "keep_first": keep}
    ids = [3 + t % 80 for t in range(length)]
    ids[reads], ids[key] = 1, 2                                           # two tokens that stand nowhere else
    return config, m, point_at(config, make_weights(config, 3), ids, reads, key), ids


@pytest.mark.parametrize("kind,window,keep,page", [("diff", 1, 0, 4), ("diff", 16, 0, 4), ("diff", 25, 0, 16), ("diff", 33, 0, 16),
                                                  ("par", 2, 1, 4), ("par", 16, 4, 4), ("par", 25, 6, 16), ("par", 9, 16, 16), ("par", 20, 33, 4)])
def test_a_key_just_inside_and_just_outside_every_edge(tmp_path, kind, window, keep, page):
    """The best key by far lies at an edge's last seen place, and one place further: the first query's logits hang on it, the
    second's must not know of it; in a prompt, decoded, in portions, at page borders and inside pages."""
    reads, shown = 60, {}
    for name, key, change in edge_cases(kind, window, keep, reads):
        config, m, weights, ids = pointed(kind, window, keep, reads, key, 70)
        folder = make_folder(tmp_path / name.replace(" ", "_"), "edge", config=config, weights=weights)
        want = {"r": exact_logits(folder, ids)}
        if change.get("size", 1):
            other = copy.deepcopy(config)
            (other["layers"][0]["mixer"] if kind == "diff" else other["layers"][0]["mixer"]["left"])["mask"].update(change)
            shown[name] = float((plain.forward(weights, other, ids).float()[reads] - want["r"][reads]).abs().max())
        r = Replayer(str(folder), "float32", 96, device="cpu", kernels=RefKernels(), page_size=page)
        for cut in ([70], [50] + [1] * 20, [7, 2, 31, 30]):
            parts = portions(ids, cut)
            compare(run(r, [([("r", p)], ["r"] if i == len(parts) - 1 else []) for i, p in enumerate(parts)]), want, "float32")
    assert shown and all(v > 0.05 for v in shown.values()), shown         # an edge one token off would show in that row


def test_pages_before_the_window_are_given_back_and_kept_ones_stay(tmp_path):
    config = copy.deepcopy(CONFIGS["par"])
    folder = make_folder(tmp_path, "par", seed=4)
    ids = random_prompt(config["vocab"], 150, 5)
    want = {"r": exact_logits(folder, ids)}
    r = Replayer(str(folder), "float32", 152, device="cpu", kernels=RefKernels(), page_size=4)
    steps = [([("r", ids[:6])], [])] + [([("r", [t])], []) for t in ids[6:]]
    compare(run(r, steps), want, "float32")
    group = r.built.cache.groups[0]
    assert group.kept == 3 and len(group.held(r.slots["r"])) <= 3 + 25 // 4 + 2
    assert r.built.cache.free_tokens() >= 152 - 12 - 25 - 8


def test_greedy_generation_through_the_scheduler(model):
    """The engine's own entry point and scheduler: greedy tokens equal the plain implementation's arg max, token by token, for
    requests that arrive together, share three slots and are cut into portions by a small step budget."""
    from holon_b200.engine import Engine, EngineConfig, SamplingParams
    folder, config, prompts, _ = model
    stored, weights = read_folder(folder)
    engine = Engine(EngineConfig(model=str(folder), dtype="float32", device="cpu", page_size=4, max_seqs=3, max_model_len=64,
                                 max_step_tokens=16, state_memory=1 << 22, prefix_cache=True, cuda_graphs=False),
                    kernels=RefKernels())
    asked = [prompts["r0"], prompts["r2"], prompts["r0"][:12] + prompts["r1"][:7], prompts["r3"]]
    with torch.inference_mode():
        got = engine.generate(asked, SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True))
    for prompt, tokens in zip(asked, got):
        ids = list(prompt)
        for token in tokens:
            logits = plain.forward(weights, stored, ids)[-1]
            best = int(logits.argmax())
            second = float(logits.topk(2).values[1])
            assert token == best or float(logits[best]) - second < 1e-3, (len(ids), token, best)
            ids.append(token)


def test_the_command_line(tmp_path, capsys):
    from holon_b200 import cli
    config = tmp_path / "config.json"
    config.write_text(json.dumps(CONFIGS["a"]))
    assert cli.main(["random-model", str(config), str(tmp_path / "m"), "--seed", "3"]) == 0
    folder = capsys.readouterr().out.strip()
    _, weights = read_folder(folder)
    assert set(weights) == {name for name, _ in tensor_table(CONFIGS["a"])}
    assert cli.main(["models"]) == 0
    assert "Bukuvik" in capsys.readouterr().out.split()


# ---------------------------------------------------------------- faults planted in the kernel table are noticed
class _Planted(RefKernels):
    """The plain kernel table with one fault; `fault` names it."""

    def __init__(self, fault: str) -> None:
        self.fault = fault

    def attention_maps(self, out, q, kv, block_table, rows, scale, cap, window, keep_first, diff, eps, gate):
        f = self.fault
        window += {"the window is one more": 1, "the window is one less": -1}.get(f, 0)
        keep_first += {"one more token is kept": 1, "one token less is kept": -1}.get(f, 0) if keep_first else 0
        if f == "the cap is left out":
            cap = None
        if f == "the gate is left out":
            gate = None
        if diff is not None:
            diff = {"the second map is left out": (0.0, diff[1]), "lambda is the constant": (diff[1], diff[1]),
                    "the factor of the difference is left out": (diff[0], 0.0)}.get(f, diff)
        super().attention_maps(out, q, kv, block_table, rows, scale, cap, window, keep_first, diff, eps, gate)

    def qkv_maps_prepare(self, q_out, kv, first, q_weight, k_weight, eps, norm, *rest):
        if self.fault == "the norm's weights are left out" and q_weight is not None:
            q_weight, k_weight = torch.ones_like(q_weight), torch.ones_like(k_weight)
        if self.fault == "q and k are not normed behind the rotation" and norm == "after":
            norm = None
        super().qkv_maps_prepare(q_out, kv, first, q_weight, k_weight, eps, norm, *rest)

    def out_norm_pair_add(self, dst, src, pair, weight, eps, offset, cast=None):
        if self.fault == "the sides' weights are swapped":
            pair.a_weight, pair.b_weight = pair.b_weight, pair.a_weight
        super().out_norm_pair_add(dst, src, pair, weight, eps, offset, cast=cast)

    def embed_pair(self, out, table, scale, *rest):
        super().embed_pair(out, table, 1.0 if self.fault == "the embedding is not scaled" else scale, *rest)

    def activation(self, x, act, numbers=None):
        super().activation(x, act, numbers)
        if self.fault == "relu without the square":
            x.copy_(x.sqrt())

    def recurrent_scan(self, out, qk, v, decay, head_decay, beta, state, rows, token_decay=None, rate=None, take=None, skip=None):
        kept = state.clone()
        if self.fault == "the step size is left out of the write":
            take = torch.ones_like(take)
        if self.fault == "the skip is left out":
            skip = torch.zeros_like(skip)
        super().recurrent_scan(out, qk, v, decay, head_decay, beta, state, rows, token_decay, rate, take, skip)
        if self.fault == "the state is not written back":
            state.copy_(kept)

    def head_norm_gate(self, out, o, weight, gate_mul, gate_pre, eps, gate="silu", gate_first=False):
        super().head_norm_gate(out, o, weight, gate_mul, gate_pre, eps, gate, gate_first and self.fault != "the gate comes behind the norm")

    def state_space_prepare(self, cb, v, dt, decay, first, at, conv, conv_bias, conv_state, dt_bias, rate_log, rows):
        kept = conv_state.clone() if conv_state is not None else None
        if self.fault == "the convolution's bias is left out":
            conv_bias = torch.zeros_like(conv_bias)
        super().state_space_prepare(cb, v, dt, decay, first, at, conv, conv_bias, conv_state, dt_bias, rate_log, rows)
        if self.fault == "B and C are swapped":
            cb.copy_(cb.flip(1))
        if self.fault == "one-token rows do not carry their inputs" and kept is not None:
            conv_state.copy_(kept)

    def conv_carry(self, conv_state, first, channels, taps, rows, least=0, at=0):
        if self.fault != "portions do not carry their inputs":
            super().conv_carry(conv_state, first, channels, taps, rows, least=least, at=at)


FAULTS = ("the window is one more", "the window is one less", "one more token is kept", "one token less is kept", "the cap is left out",
          "the gate is left out", "the second map is left out", "lambda is the constant", "the norm's weights are left out",
          "q and k are not normed behind the rotation", "the sides' weights are swapped", "the embedding is not scaled",
          "relu without the square", "the step size is left out of the write", "the skip is left out", "the state is not written back",
          "the gate comes behind the norm", "the convolution's bias is left out", "B and C are swapped",
          "one-token rows do not carry their inputs", "portions do not carry their inputs")


def test_planted_faults_are_noticed(tmp_path):
    """Portions beside single tokens of three requests of configuration `a`, in 32-bit: the comparison accepts the plain kernel
    table and rejects every table with one fault planted (YaRN, the layer scale and the residual multiplier are planted in the
    configuration and the weights)."""
    folder = make_folder(tmp_path, "a", seed=7)
    config = CONFIGS["a"]
    prompts = {f"r{i}": random_prompt(config["vocab"], n, 60 + i) for i, n in enumerate((23, 41, 30))}
    want = {rid: exact_logits(folder, ids) for rid, ids in prompts.items()}
    cut = {rid: portions(ids, sizes) for (rid, ids), sizes in zip(prompts.items(), ([5, 1, 1, 3], [2, 9, 1], [30]))}
    steps = []
    for j in range(max(len(p) for p in cut.values())):
        steps.append(([(rid, p[j]) for rid, p in cut.items() if j < len(p)], [rid for rid, p in cut.items() if j == len(p) - 1]))

    def missed_by(where, kernels):
        try:
            compare(run(Replayer(str(where), "float32", 192, device="cpu", kernels=kernels, page_size=64), steps), want, "float32")
            return True
        except AssertionError:
            return False

    assert missed_by(folder, RefKernels())
    missed = [fault for fault in FAULTS if missed_by(folder, _Planted(fault))]
    stored, weights = read_folder(folder)
    changes = [({("layers", 1, "mixer", "left", "rot", "scaling", "factor"): 1.0}, {}),
               ({("layers", 1, "mixer", "left", "rot", "scaling", "original"): 4096}, {}),
               ({("residual_mult",): 1.0}, {}), ({("layers", 0, "mixer", "diff"): 0.5}, {}),
               ({}, {"l1.ls1": torch.ones_like(weights["l1.ls1"])}), ({}, {"l0.ls2": weights["l0.ls1"].clone()})]
    for i, (paths, tensors) in enumerate(changes):
        other = copy.deepcopy(stored)
        for path, value in paths.items():
            at = other
            for key in path[:-1]:
                at = at[key]
            at[path[-1]] = value
        if missed_by(make_folder(tmp_path / str(i), "a", config=other, weights={**weights, **tensors}), RefKernels()):
            missed.append(f"change {i}")
    assert not missed, f"the comparison accepted: {missed}"

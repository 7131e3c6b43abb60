"""Gegunex without a GPU: configuration, weight names, each new kernel twin against the written-out rule, and the engine's
host side (batch layout, cache entries with windows, the per-request state of the matrix-state layers) with the CPU twins of
the kernels (tests/ref_kernels.py) against the plain implementation (tests/plain_gegunex.py)."""
from __future__ import annotations

import copy
import json
import math

import pytest
import torch

import plain_gegunex as plain
from gegunex_tools import CONFIGS, compare, exact_logits, make_folder, make_weights, point_at, read_folder, stored_config, tensor_table
from helpers import random_prompt
from holon_b200.config.registry import ConfigError, resolve_architecture
from holon_b200.replay import Replayer
from ref_kernels import RefKernels
from replay_tools import portions, run


def test_architecture_and_configuration():
    arch = resolve_architecture(CONFIGS["a"])
    cfg = arch.parse(CONFIGS["a"])
    assert arch.name == "Gegunex" and len(cfg.layers) == 5 and cfg.layers[4].mlp is None
    spec = arch.recipe(cfg)
    assert [(r.layer, r.cache, r.fills) for r in spec.order] == [(i, i, True) for i in range(5)]
    assert all(layer.block.name == "prenorm" and layer.norm.name == "layernorm" for layer in spec.layers)
    assert spec.layers[0].block.kwargs()["residual_mult"] == 0.6 and spec.head.kwargs() == {"tied": True, "softcap": 9.0}
    assert [layer.mixer.name for layer in spec.layers] == ["gated_delta", "latent", "lightning", "latent", "gated_delta"]
    m = spec.layers[1].mixer.kwargs()
    assert (m["window"], m["q_rank"], m["rank"], m["sink"], m["gate"]) == (7, 40, 24, True, False)
    rope = m["position"].kwargs()
    assert rope["interleaved"] and rope["yarn"] == (4.0, 64.0, 8.0, 1.0) and rope["rotary_dim"] == 12
    assert spec.layers[3].mixer.kwargs()["position"].kwargs()["yarn"] is None
    f = spec.layers[1].ffn.kwargs()
    assert (f["experts"], f["top"], f["inter"], f["limit"], f["scores"], f["weight_on"]) == (6, 3, 24, 0.8, "sigmoid", "input")
    for path, value, error in (
            (("layers", 0, "type"), "retention", NotImplementedError),
            (("layers", 0, "mlp", "kind"), "dense", NotImplementedError),
            (("layers", 0, "mixer", "kv_heads"), 3, ConfigError),
            (("layers", 0, "mixer", "conv"), 0, ConfigError),
            (("layers", 1, "mixer", "rot", "dims"), 14, ConfigError),
            (("layers", 1, "mixer", "rot", "dims"), 5, ConfigError),
            (("layers", 1, "mixer", "rot", "scaling", "factor"), 0.0, ConfigError),
            (("layers", 1, "mixer", "rot", "scaling"), {"factor": 2.0}, ConfigError),
            (("layers", 1, "mixer", "mask", "size"), 0, ConfigError),
            (("layers", 1, "mixer", "q_rank"), 0, ConfigError),
            (("layers", 1, "mlp", "router", "top"), 7, ConfigError),
            (("layers", 1, "mlp", "expert", "limit"), -1.0, ConfigError),
            (("layers", 2, "mixer", "decay"), [0.5, 0.9], ConfigError),
            (("logit_softcap",), 0.0, ConfigError),
            (("width",), 0, ConfigError)):
        c = copy.deepcopy(CONFIGS["a"])
        at = c
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(error):
            arch.parse(c)
    c = copy.deepcopy(CONFIGS["a"])
    del c["layers"][1]["mixer"]["mask"]
    assert arch.parse(c).layers[1].mixer.window == 0                        # no mask: every earlier token is seen
    with pytest.raises(ConfigError):                                       # the ranks come from a dict or from shapes
        arch.parse(stored_config(CONFIGS["a"]))
    done = arch.complete(stored_config(CONFIGS["a"]), {"l0.mix.a1": (6, 64), "l0.mix.g1": (5, 64), "l4.mix.a1": (4, 64), "l4.mix.g1": (4, 64)})
    assert arch.parse(done) == cfg


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
    del tensors["l1.mix.sink"]
    tensors["l1.mix.dq.norm"] = torch.zeros(3, dtype=torch.bfloat16)
    tensors["l4.norm2"] = tensors["l0.norm2"].clone()                     # layer 4 has no feed-forward
    save_file(tensors, str(folder / "model.safetensors"))
    with pytest.raises(WeightError) as e:
        Replayer(str(folder), "float32", 64, device="cpu", kernels=RefKernels())
    assert e.value.missing == ["l1.mix.sink"] and e.value.unexpected == ["l4.norm2"]
    assert [s[0] for s in e.value.shapes] == ["l1.mix.dq.norm"]


# ---------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("base,dims,scaling", [(300.0, 12, (4.0, 64, 8.0, 1.0)), (1e6, 64, (32.0, 4096, 32.0, 1.0)), (50.0, 2, (2.0, 32, 4.0, 0.5)),
                                               (10.0, 8, (1.0, 16, 2.0, 2.0)), (500.0, 20, (8.0, 8, 64.0, 32.0)), (1e4, 16, None)])
def test_rotation_tables(base, dims, scaling):
    """Frequencies and the factor on cosines and sines, over ramps that begin below the first pair, end past the last,
    and have no width."""
    from holon_b200.parts.base import BuildContext
    from holon_b200.parts.position import Rope
    rot = {"base": base, "dims": dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    freq, size = plain.frequencies(rot)
    table = Rope(BuildContext("cpu", torch.float32, None, max_positions=90), theta=base, rotary_dim=dims, head_dim=dims, interleaved=True,
                 yarn=scaling).table.double()
    angle = torch.arange(90, dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)[None]
    assert torch.allclose(table, torch.cat((angle.cos(), angle.sin()), -1) * size, atol=3e-5)
    if scaling and scaling[0] != 1.0:
        assert abs(size - (0.1 * math.log(scaling[0]) + 1)) < 1e-12 and min(freq) < base ** (-2.0 * (dims // 2 - 1) / dims) + 1e-12


def test_layer_norm_with_a_factor_and_rows_of_pairs():
    k = RefKernels()
    g = torch.Generator().manual_seed(3)
    h, y = torch.randn(5, 24, generator=g) + 2.0, torch.randn(15, 24, generator=g)
    w, place = 1 + 0.2 * torch.randn(24, generator=g), torch.randperm(15, generator=g).to(torch.int32)
    want = h.double() + 0.7 * torch.stack([y[place[3 * t:3 * t + 3].long()].double().sum(0) for t in range(5)])
    normed = plain.layer_norm(want, w.double(), 1e-5)
    out, hh = torch.empty(5, 24), h.clone()
    k.add_layernorm(out, hh, y, 0.7, w, 1e-5, None, place=place)
    assert torch.allclose(out.double(), normed, atol=1e-5) and torch.allclose(hh.double(), want, atol=1e-6)
    index = torch.tensor([4, 1], dtype=torch.int32)
    out, hh = torch.empty(2, 24), h.clone()
    k.add_layernorm(out, hh, y, 0.7, w, 1e-5, index, place=place)
    assert torch.allclose(out.double(), normed[[4, 1]], atol=1e-5) and torch.equal(hh, h)


def test_a_stream_with_pairs_and_a_factor_under_another_norm():
    """A norm that takes neither gets the pending output added up and scaled first."""
    from holon_b200.parts.base import BuildContext, PairRows, Residual
    from holon_b200.parts.norm import RMSNorm
    ctx = BuildContext("cpu", torch.float32, RefKernels(), max_positions=8)
    norm = RMSNorm(ctx, eps=1e-5, dim=8)
    norm.weight.tensor = torch.ones(8)
    h, y, place = torch.randn(3, 8), torch.randn(6, 8), torch.tensor([3, 0, 5, 1, 2, 4], dtype=torch.int32)
    want = h + 0.5 * torch.stack([y[3] + y[0], y[5] + y[1], y[2] + y[4]])
    for index in (None, torch.tensor([2], dtype=torch.int32)):
        stream = Residual(h.clone(), PairRows(ctx, y, place, 3))
        stream.delta_scale = 0.5
        out = norm.add(stream) if index is None else stream.final_rows(norm, index)
        rows = want if index is None else want[index.long()]
        assert torch.allclose(out, plain.rms_norm(rows, torch.ones(8), 1e-5), atol=1e-5)
        assert torch.allclose(stream.h, want, atol=1e-6) and stream.delta is None and stream.delta_scale == 1.0


def test_experts_against_the_written_out_rule():
    """The choice by sigmoid scores, the weight ahead of the limits (a weight on the output would land elsewhere), the
    limits themselves reached on both sides."""
    from holon_b200.config.spec import PartRef
    from holon_b200.parts.base import BuildContext
    k, (experts, top, ff, width, limit) = RefKernels(), (5, 3, 12, 16, 0.6)
    ctx = BuildContext("cpu", torch.float32, k, max_positions=8)
    part = ctx.part(PartRef.of("ffn", "experts", experts=experts, top=top, scale=1.0, inter=ff, activation="clamped", gated=True,
                               limit=limit, scores="sigmoid", weight_on="input"), hidden=width)
    g = torch.Generator().manual_seed(9)
    weights = {}
    for name, p, (r0, r1) in part.loadables():
        if p.tensor is None:
            p.tensor = torch.empty(p.shape)
        weights[name] = 2.5 * torch.randn(p.piece_shape((r0, r1)), generator=g) / p.shape[1] ** 0.5
        p.tensor[r0:r1] = weights[name]
    x = torch.randn(7, width, generator=g)
    mlp = {"expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    want = plain.experts_ff(x.double(), weights, "", mlp)
    assert torch.allclose(part.forward(x, None).double(), want, atol=1e-5)
    assert torch.allclose(part.forward(x, None, pairs=True).combined().double(), want, atol=1e-5)
    z = x.double() @ weights["router"].double().T
    other = torch.zeros_like(want)
    for t in range(7):
        for e, share in plain.choose(z[t], top):
            other[t] += share * plain.clamped_unit(x[t].double(), weights, f"e{e}.", limit)
    assert float((other - want).abs().max()) > 0.05


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
    paged = [i for i, layer in enumerate(config["layers"]) if layer["type"] == "latent_attention"]
    assert sorted(e for g in r.built.cache.groups for e in g.entries) == paged
    states = r.built.cache.slot_states
    for i, layer in enumerate(config["layers"]):
        m = layer["mixer"]
        if layer["type"] == "latent_attention":                          # the latent and the shared rotated part, nothing per head
            assert tuple(r.built.cache.group_of_entry[i].kv.shape[2:]) == (4, m["kv_rank"] + m["rot_dim"])
            assert not [key for key in states if key[0] == i]
            continue
        s = states[(i, "state")]
        assert tuple(s.shape[1:]) == (m["heads"], m["vdim"], m["dim"]) and s.dtype == torch.float32
        if m.get("conv", 1) > 1:
            assert tuple(states[(i, "conv")].shape[1:]) == (m["conv"] - 1, 2 * m["kv_heads"] * m["dim"] + m["heads"] * m["vdim"])
        else:
            assert (i, "conv") not in states
    assert all(s.shape[0] == 5 for s in states.values())                  # four requests and the padding slot


def test_whole_tail_portions_and_mixed(model):
    folder, config, prompts, want = model
    r = Replayer(str(folder), "float32", 64, device="cpu", kernels=RefKernels(), page_size=4)
    compare(run(r, [([(rid, ids)], [rid]) for rid, ids in prompts.items()]), want, "float32")
    steps = []
    for rid, ids in prompts.items():                                       # a portion, then one by one
        steps.append(([(rid, ids[:5])], []))
        steps += [([(rid, [t])], [rid] if i == len(ids) - 6 else []) for i, t in enumerate(ids[5:])]
    compare(run(r, steps), want, "float32")
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
    # again (a slot's matrix state, its carried inputs and its pages must not leak into the request that takes it next)
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
        assert torch.allclose(alone[("r1", pos)], both[("r1", pos)], atol=5e-5, rtol=0)


def pointed_model(window, distance, length=70, reads=60):
    """A single latent layer with a window, built so that the query at `reads` puts nearly all its weight on the key
    `distance` places before it, if it sees that key: (configuration, weights, ids)."""
    config = copy.deepcopy(CONFIGS["lat"])
    config["layers"][0]["mixer"]["mask"]["size"] = window
    ids = [3 + t % 80 for t in range(length)]
    ids[reads], ids[reads - distance] = 1, 2                              # two tokens that stand nowhere else
    weights = make_weights(config, 3)
    return config, point_at(config, weights, 0, ids, reads, reads - distance, 12.0), ids


@pytest.mark.parametrize("page", [4, 16])
@pytest.mark.parametrize("window", [1, 2, 16, 25, 33])
def test_a_key_just_inside_and_just_outside_the_window(tmp_path, window, page):
    """The best key by far lies at the window's last seen place, and one place further back: the first query's logits
    hang on it, the second's must not know of it; in a prompt and decoded, at page borders and inside pages."""
    reads = 60
    seen = {}
    for inside in (True, False):
        distance = window - 1 if inside else window
        config, weights, ids = pointed_model(window, distance) if distance else pointed_model(window, 1)
        folder = make_folder(tmp_path / str(inside), "edge", config=config, weights=weights)
        want = {"r": exact_logits(folder, ids)}
        if distance:
            wide = copy.deepcopy(config)
            wide["layers"][0]["mixer"]["mask"]["size"] = window + (-1 if inside and window > 1 else 1)
            moved = plain.forward(weights, wide, ids).float()
            seen[inside] = float((moved[reads] - want["r"][reads]).abs().max())
        r = Replayer(str(folder), "float32", 96, device="cpu", kernels=RefKernels(), page_size=page)
        compare(run(r, [([("r", ids)], ["r"])]), want, "float32")
        steps = [([("r", ids[:50])], [])] + [([("r", [t])], ["r"] if i == len(ids) - 51 else []) for i, t in enumerate(ids[50:])]
        compare(run(r, steps), want, "float32")
        parts = portions(ids, [7, 2, 31])
        compare(run(r, [([("r", p)], ["r"] if i == len(parts) - 1 else []) for i, p in enumerate(parts)]), want, "float32")
    assert all(v > 0.05 for v in seen.values()), seen                      # a window one token off would show in that row


def test_pages_before_the_window_are_given_back(tmp_path):
    """300 tokens decoded through a pool that holds far fewer: what lies before every window is given back and used again."""
    config = copy.deepcopy(CONFIGS["lat"])
    folder = make_folder(tmp_path, "lat", seed=4)
    ids = random_prompt(config["vocab"], 200, 5)
    want = {"r": exact_logits(folder, ids)}
    r = Replayer(str(folder), "float32", 200, device="cpu", kernels=RefKernels(), page_size=4)
    steps = [([("r", ids[:6])], [])] + [([("r", [t])], []) for t in ids[6:]]
    compare(run(r, steps), want, "float32")
    assert r.built.cache.free_tokens() >= 200 - 25 - 8


def test_greedy_generation_through_the_scheduler(model):
    """The engine's own entry point and scheduler: greedy tokens equal the plain implementation's arg max, token by
    token, for requests that arrive together, share three slots and are cut into portions by a small step budget."""
    from holon_b200.engine import Engine, EngineConfig, SamplingParams
    folder, config, prompts, _ = model
    stored, weights = read_folder(folder)
    engine = Engine(EngineConfig(model=str(folder), dtype="float32", device="cpu", page_size=4, max_seqs=3, max_model_len=64,
                                 max_step_tokens=16, state_memory=1 << 22, prefix_cache=True, cuda_graphs=False),
                    kernels=RefKernels())
    asked = [prompts["r0"], prompts["r2"], prompts["r0"][:12] + prompts["r1"][:7], prompts["r3"]]
    with torch.inference_mode():
        got = engine.generate(asked, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
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
    assert "Gegunex" in capsys.readouterr().out.split()


# ---------------------------------------------------------------- faults planted in the kernel table are noticed
class _Planted(RefKernels):
    """The plain kernel table with one fault; `fault` names it."""

    def __init__(self, fault: str) -> None:
        self.fault = fault

    def latent_attention(self, out, qa, cache, block_table, rows, scale, rank, window, sinks=None):
        if self.fault == "the sink is left out":
            sinks = None
        if self.fault == "the sink is scaled":
            sinks = sinks * scale
        window += {"the window is one more": 1, "the window is one less": -1}.get(self.fault, 0)
        super().latent_attention(out, qa, cache, block_table, rows, scale, rank, window, sinks=sinks)

    def latent_prepare(self, *args, interleaved=False, cq=None, cq_at=0, cq_weight=None):
        if self.fault == "halves turn instead of neighbours":
            interleaved = False
        if self.fault == "the query latent's weight is left out" and cq is not None:
            cq_weight = torch.ones_like(cq_weight)
        super().latent_prepare(*args, interleaved=interleaved, cq=cq, cq_at=cq_at, cq_weight=cq_weight)

    def add_layernorm(self, out, h, delta, scale, weight, eps, index, place=None):
        if self.fault == "the residual multiplier is left out":
            scale = 1.0
        super().add_layernorm(out, h, delta, scale, weight, eps, index, place=place)
        if self.fault == "the mean stays in":
            x = h if index is None else h[index.long()]
            if index is None or delta is None:
                self.rmsnorm(out, x, weight, eps, 0.0)

    def softcap(self, x, cap):
        if self.fault != "the logits' limit is left out":
            super().softcap(x, cap)

    def retention_prepare(self, qk, v, first, positions, table, rot_dims, k_scale, silu=False):
        super().retention_prepare(qk, v, first, positions, table, rot_dims, k_scale,
                                  silu=silu and self.fault != "q, k and v pass no silu")

    def head_norm_gate(self, out, o, weight, gate_mul, gate_pre, eps, gate="silu"):
        if self.fault == "each head is normed alone" and o.shape[1] == 1 and gate_pre is not None:
            o = o.view(o.shape[0], -1, 20)
            y = o * torch.rsqrt((o * o).mean(-1, keepdim=True) + eps)
            out.copy_((y.reshape(out.shape) * weight * torch.sigmoid(gate_pre.reshape(out.shape))).to(out.dtype))
            return
        super().head_norm_gate(out, o, weight, gate_mul, gate_pre, eps, gate=gate)

    def recurrent_scan(self, out, qk, v, decay, head_decay, beta, state, rows, token_decay=None, rate=None):
        kept = state.clone()
        super().recurrent_scan(out, qk, v, decay, head_decay, beta, state, rows, token_decay, rate)
        if self.fault == "the state is not written back":
            state.copy_(kept)

    def delta_prepare(self, *args, carry=False):
        super().delta_prepare(*args, carry=carry and self.fault != "one-token rows do not carry their inputs")

    def conv_carry(self, conv_state, first, channels, taps, rows, least=0):
        if self.fault != "portions do not carry their inputs":
            super().conv_carry(conv_state, first, channels, taps, rows, least=least)

    def route_rows(self, *args, scores="softmax", row_weight=None, **kw):
        if self.fault == "the scores are shares of a softmax":
            scores = "softmax"
        super().route_rows(*args, scores=scores, row_weight=row_weight, **kw)
        if self.fault == "the chosen weights are renormalized":
            weight, place = args[1], args[3]
            row_weight[place.long()] = (weight / weight.sum(-1, keepdim=True)).reshape(-1)

    def expert_glu(self, out, x, token_of, w, starts, limit, alpha, row_scale):
        if self.fault == "the experts read their input unweighted":
            row_scale = None
        if self.fault == "the limit is left out":
            limit = 1e9
        super().expert_glu(out, x, token_of, w, starts, limit, alpha, row_scale)


FAULTS = ("the sink is left out", "the sink is scaled", "the window is one more", "the window is one less",
          "halves turn instead of neighbours", "the query latent's weight is left out", "the residual multiplier is left out",
          "the mean stays in", "the logits' limit is left out", "q, k and v pass no silu", "each head is normed alone",
          "the state is not written back", "one-token rows do not carry their inputs", "portions do not carry their inputs",
          "the scores are shares of a softmax", "the chosen weights are renormalized", "the experts read their input unweighted",
          "the limit is left out")


def test_planted_faults_are_noticed(tmp_path):
    """Portions beside single tokens of three requests of configuration `a`, in 32-bit: the comparison accepts the plain
    kernel table and rejects every table with one fault planted (YaRN left out, or its factor on cosines and sines, is
    planted in the configuration)."""
    folder = make_folder(tmp_path, "a", seed=7)
    config = CONFIGS["a"]
    prompts = {f"r{i}": random_prompt(config["vocab"], n, 60 + i) for i, n in enumerate((23, 41, 30))}
    want = {rid: exact_logits(folder, ids) for rid, ids in prompts.items()}
    cut = {rid: portions(ids, sizes) for (rid, ids), sizes in zip(prompts.items(), ([5, 1, 1, 3], [2, 9, 1], [30]))}
    steps = []
    for j in range(max(len(p) for p in cut.values())):
        steps.append(([(rid, p[j]) for rid, p in cut.items() if j < len(p)], [rid for rid, p in cut.items() if j == len(p) - 1]))

    def replay(where, kernels):
        return run(Replayer(str(where), "float32", 128, device="cpu", kernels=kernels, page_size=4), steps)

    compare(replay(folder, RefKernels()), want, "float32")
    missed = []
    for fault in FAULTS:
        try:
            compare(replay(folder, _Planted(fault)), want, "float32")
            missed.append(fault)
        except AssertionError:
            pass
    stored, weights = read_folder(folder)
    for change in ({"factor": 1.0}, {"original": 4096}):
        other = copy.deepcopy(stored)
        other["layers"][1]["mixer"]["rot"]["scaling"].update(change)
        try:
            compare(replay(make_folder(tmp_path / str(change), "a", config=other, weights=weights), RefKernels()), want, "float32")
            missed.append(f"YaRN with {change}")
        except AssertionError:
            pass
    assert not missed, f"the comparison accepted: {missed}"

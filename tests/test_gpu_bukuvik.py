"""Bukuvik on the GPU. Each new or extended kernel alone against its plain twin (tests/ref_kernels.py) or the rule written out in
64-bit, with inputs made so that a fault shows (one key that takes all the weight just inside or outside an edge, scores that the
cap bends and scores it hardly touches, two maps that nearly cancel, large row means, step sizes from near 0 to several units);
then the replayer in 32-bit and bfloat16 against the plain implementation (tests/plain_bukuvik.py): whole prompts, prefill against
token-by-token decoding, portions down to two tokens, unequal requests mixed in a pool whose pages and slots are used again, the
first tokens, long decoding, sizes that are multiples of nothing, sizes the tensor cores take; and greedy generation through the
engine's scheduler and graphs."""
from __future__ import annotations

import copy
import types

import pytest
import torch

import plain_bukuvik as plain
from bukuvik_tools import CONFIGS, _att, _diff, _model, _par, _rot, _ssm, compare, exact_logits, make_folder, make_weights, point_at, read_folder
from helpers import random_prompt
from holon_b200.replay import Replayer
from ref_kernels import RefKernels
from replay_tools import mixed_trace, portions, run

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
REF = RefKernels()
F64 = torch.float64


@pytest.fixture(scope="module")
def K():
    from holon_b200.kernels import load_kernels
    return load_kernels(DEV)


def rand(*shape, dtype=torch.float32, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def close(got, want, dtype, scale=1.0):
    tol = (3e-5 if dtype == torch.float32 else 1.6e-2) * scale
    diff = (got.float().cpu() - want.float().cpu()).abs().max().item()
    assert diff <= tol, f"difference {diff} > {tol}"


def rows_of(counts, slots, kv_len=None, device=DEV):
    """The rows of a step: `counts` tokens each, in slots `slots`, holding `kv_len` tokens after the step."""
    qs = [0]
    for n in counts:
        qs.append(qs[-1] + n)
    t = lambda x: torch.tensor(x, dtype=torch.int32, device=device)      # noqa: E731
    kv = kv_len or counts
    return types.SimpleNamespace(query_start=t(qs), row_slot=t(slots), kv_len=t(kv), n_rows=len(counts), n_tokens=qs[-1],
                                 n_decode=sum(1 for n in counts if n == 1), max_q=max(counts), max_kv=max(kv),
                                 host_query_start=qs, host_kv_len=kv, plan={})


# ---------------------------------------------------------------- the norm on an output, alone and for a pair
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,dim", [(7, 64), (3, 72), (5, 1030), (300, 2048), (2, 33), (9, 3000), (4, 4096), (2, 8192), (2, 12288), (3, 11903)])
@pytest.mark.parametrize("weight32", [False, True])
def test_norm_of_a_pair_and_of_one_output(K, dtype, rows, dim, weight32):
    from holon_b200.parts.base import NormedPair
    src, a, b = rand(rows, dim, seed=1), rand(rows, dim, dtype=dtype, seed=2, scale=3.0), rand(rows, dim, dtype=dtype, seed=3, scale=0.2) + 1.0
    b = b.to(dtype)
    wa, wb, w = ((1 + 0.3 * rand(dim, seed=s)).to(torch.float32 if weight32 else dtype) for s in (4, 5, 6))
    unit = lambda y, e: y * torch.rsqrt((y * y).mean(-1, keepdim=True) + e)      # noqa: E731
    z = 0.5 * (unit(a.to(F64), 1e-5) * wa.to(F64) + unit(b.to(F64), 1e-5) * wb.to(F64))
    for one in (False, True):
        want = src.to(F64) + unit(a.to(F64) if one else z, 1e-6) * (w.to(F64) + 0.25)
        for in_place in (False, True):
            s = src.to(DEV)
            dst = s if in_place else torch.empty_like(s)
            cast = torch.empty(rows, dim, dtype=dtype, device=DEV)
            if one:
                K.out_norm_add(dst, s, a.to(DEV), None, w.to(DEV), 1e-6, 0.25, cast=cast)
            else:
                K.out_norm_pair_add(dst, s, NormedPair(a.to(DEV), wa.to(DEV), b.to(DEV), wb.to(DEV), 1e-5, 0.5), w.to(DEV), 1e-6, 0.25, cast=cast)
            close(dst, want, torch.float32)
            close(cast, want, dtype, scale=2.0)
    dst = torch.empty(rows, dim, device=DEV)
    K.out_norm_pair_add(dst, src.to(DEV), NormedPair(a.to(DEV), wa.to(DEV), b.to(DEV), wb.to(DEV), 1e-5, 0.5), w.to(DEV), 1e-6, 0.25)
    close(dst, src.to(F64) + unit(z, 1e-6) * (w.to(F64) + 0.25), torch.float32)


# ---------------------------------------------------------------- the squared relu in the first product
@pytest.mark.parametrize("m,n,k", [(1, 96, 64), (8, 20000, 64), (9, 330, 256), (16, 48, 40), (20, 520, 128), (32, 100, 72), (100, 256, 64), (150, 1000, 320),
                                   (300, 513, 128), (2048, 640, 512), (7000, 64, 64), (40, 64, 64), (5, 50, 33)])
@pytest.mark.parametrize("pair", [True, False])
def test_squared_relu_in_the_product(K, m, n, k, pair, monkeypatch):
    monkeypatch.setattr(K, "gemm_pair", pair)
    x, w = rand(m, k, dtype=torch.bfloat16, seed=1), rand(n, k, dtype=torch.bfloat16, seed=2, scale=k ** -0.5)
    out = torch.full((m, n), float("nan"), dtype=torch.bfloat16, device=DEV)
    took = K.linear_relu2(out, x.to(DEV), w.to(DEV))
    assert took == (k % 8 == 0 and (m <= 32 or 96 < m <= 6144))
    if took:
        want = torch.relu(x.to(F64) @ w.to(F64).T) ** 2
        d = (out.cpu().to(F64) - want).abs()
        assert bool((d <= 2 ** -8 * want + 1e-4).all())
        assert K.tcgen05_status() == 0


# ---------------------------------------------------------------- state space
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,groups,n,vdim,taps", [(6, 3, 40, 20, 3), (4, 4, 16, 8, 4), (3, 1, 7, 5, 1), (5, 5, 3, 2, 6), (8, 1, 128, 64, 4), (2, 1, 130, 33, 2)])
def test_state_space_inputs_and_carried_rows(K, dtype, heads, groups, n, vdim, taps):
    """Portions and one-token rows of three requests, twice in a row (the second step reads what the first carried)."""
    inner, channels = heads * vdim, heads * vdim + 2 * groups * n
    conv, bias = rand(channels, taps, dtype=dtype, seed=1, scale=0.6), rand(channels, dtype=dtype, seed=2)
    dt_bias, rate = rand(heads, seed=3, scale=4.0), rand(heads, seed=4, scale=1.5)
    state = rand(5, max(1, taps - 1), channels, dtype=dtype, seed=5)[:, :taps - 1]
    states = {d: state.clone().to(d) for d in ("cpu", DEV)} if taps > 1 else {"cpu": None, DEV: None}
    for step, counts in enumerate(([1, 1, 9], [1, 2, 3], [1, 1, 1])):
        t = sum(counts)
        first = rand(t, inner + channels + heads, dtype=dtype, seed=10 + step, scale=1.5)
        got = {}
        for device, k in (("cpu", REF), (DEV, K)):
            rows = rows_of(counts, [3, 0, 2], device=device)
            out = [torch.full(s, float("nan"), device=device) for s in ((t, 2, groups, n), (t, heads, vdim), (t, heads), (t, heads))]
            k.state_space_prepare(*out, first.to(device), inner, conv.to(device), bias.to(device), states[device], dt_bias.to(device),
                                  rate.to(device), rows)
            k.conv_carry(states[device], first.to(device), channels, taps, rows, least=2, at=inner)
            got[device] = out
        for a, b in zip(got[DEV], got["cpu"]):
            assert torch.isfinite(a).all()
            close(a, b, torch.float32, scale=1.0 + float(b.abs().max()))
        if taps > 1:
            assert torch.equal(states[DEV].cpu(), states["cpu"])


@pytest.mark.parametrize("heads,groups,n,vdim", [(4, 2, 16, 12), (3, 1, 7, 5), (8, 2, 128, 64), (2, 2, 1, 3), (2, 1, 96, 40), (4, 1, 256, 128), (2, 1, 300, 17)])
@pytest.mark.parametrize("counts", [[1, 1, 1], [37], [1, 1, 5, 200], [64, 129], [2, 63, 65, 300], [1, 513]])
def test_scan_with_step_sizes_and_skips(K, heads, groups, n, vdim, counts):
    """The scan and its form in chunks against the rule in 64-bit: step sizes from 1e-4 to several units, rates that forget at once and rates that keep
    hundreds of tokens, states that are not empty at the start."""
    t, slots = sum(counts), [4, 1, 3, 0][:len(counts)]
    cb, v = rand(t, 2, groups, n, seed=1), rand(t, heads, vdim, seed=2)
    dt = torch.exp(rand(t, heads, seed=3, scale=2.0) - 2.0)
    rate_log, skip = torch.linspace(-6.0, 1.5, heads), rand(heads, seed=5)
    decay = torch.exp(-torch.exp(rate_log) * dt)
    state0 = rand(6, heads, vdim, n, seed=6)
    want, after = torch.zeros(t, heads, vdim, dtype=F64), state0.to(F64).clone()
    at = 0
    for count, slot in zip(counts, slots):
        S = after[slot].clone()                                            # [heads, vdim, n]
        for i in range(at, at + count):
            B, C = (cb[i, w].to(F64).repeat_interleave(heads // groups, 0) for w in (1, 0))
            x = v[i].to(F64)
            S = decay[i].to(F64)[:, None, None] * S + (dt[i].to(F64)[:, None] * x)[:, :, None] * B[:, None, :]
            want[i] = (S * C[:, None, :]).sum(-1) + skip.to(F64)[:, None] * x
        after[slot], at = S, at + count
    for chunks in (False, True):
        out = torch.full((t, heads, vdim), float("nan"), device=DEV)
        state = state0.to(DEV)
        if chunks:
            K.state_space_scan(out, cb.to(DEV), v.to(DEV), dt.to(DEV), decay.to(DEV), rate_log.to(DEV), skip.to(DEV), state, rows_of(counts, slots))
        else:
            K.recurrent_scan(out, cb.to(DEV), v.to(DEV), None, None, None, state, rows_of(counts, slots), token_decay=decay.to(DEV),
                             take=dt.to(DEV), skip=skip.to(DEV))
        close(out, want, torch.float32, scale=0.2 * (1.0 + float(want.abs().max())))
        close(state, after, torch.float32, scale=0.2 * (1.0 + float(after.abs().max())))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("gate", ["sigmoid", "silu"])
@pytest.mark.parametrize("parts,width", [(1, 60), (3, 20), (2, 512), (1, 640), (4, 1024), (2, 1030), (1, 11264), (1, 12288)])
def test_a_gate_ahead_of_the_norm(K, dtype, gate, parts, width):
    t, n = 7, parts * width
    y, wide, w = rand(t, parts, width, seed=1), rand(t, n + 24, dtype=dtype, seed=2, scale=2.0), 1 + 0.3 * rand(n, seed=3)
    out, want = torch.empty(t, parts, width, dtype=dtype, device=DEV), torch.empty(t, parts, width)
    K.head_norm_gate(out, y.to(DEV), w.to(DEV), None, wide.to(DEV)[:, 8:8 + n], 1e-5, gate=gate, gate_first=True)
    g = wide[:, 8:8 + n].to(F64).view(t, parts, width)
    g = torch.sigmoid(g) * (g if gate == "silu" else 1.0)
    z = y.to(F64) * g
    want = z * torch.rsqrt((z * z).mean(-1, keepdim=True) + 1e-5) * w.to(F64).view(parts, width)
    close(out, want, dtype, scale=4.0)


# ---------------------------------------------------------------- attention with one or two maps
def turn_table(dims, positions=512, base=300.0, size=1.2):
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    angle = torch.arange(positions, dtype=torch.float32)[:, None] * freq[None]
    return (torch.cat((angle.cos(), angle.sin()), -1) * size).contiguous()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("norm", [None, "before", "after"])
@pytest.mark.parametrize("heads,kv,maps,dim,vdim,rot", [(6, 2, 2, 56, 72, 24), (6, 3, 1, 96, 64, 48), (3, 1, 2, 11, 7, 4), (2, 2, 1, 17, 5, 16), (1, 1, 2, 8, 3, 0),
                                                       (32, 8, 1, 128, 128, 128), (2, 1, 2, 200, 150, 100), (2, 1, 1, 512, 64, 2)])
def test_queries_and_cache_rows(K, dtype, norm, heads, kv, maps, dim, vdim, rot):
    t, page = 9, 4
    first = rand(t, (heads * maps + kv * maps) * dim + kv * vdim + 6, dtype=dtype, seed=1, scale=2.0)
    table = turn_table(rot) if rot else None
    pos = torch.tensor([0, 1, 2, 7, 100, 511, 600, 3, 4], dtype=torch.int32)
    write = torch.tensor([0, 5, 11, 2, -1, 23, 24, 99, 7], dtype=torch.int32)      # negative, on the null page, past the pool: skipped
    wq, wk = (1 + 0.3 * rand(dim, seed=s) for s in (3, 4))
    got = {}
    for device, k in (("cpu", REF), (DEV, K)):
        q = torch.full((t, heads, maps, dim), float("nan"), dtype=dtype, device=device)
        cache = torch.zeros(7, kv, page, maps * dim + vdim, dtype=dtype, device=device)
        d = lambda x: x.to(device) if x is not None else None              # noqa: E731
        k.qkv_maps_prepare(q, cache, d(first), d(wq) if norm == "before" else None, d(wk) if norm == "before" else None, 1e-5, norm,
                           d(pos.clamp(max=511)) if device == "cpu" else d(pos), d(table), rot, d(write), kv, vdim)
        got[device] = (q, cache)
    close(got[DEV][0], got["cpu"][0], dtype, scale=4.0)
    close(got[DEV][1], got["cpu"][1], dtype, scale=4.0)
    assert float(got["cpu"][1][:6].abs().sum()) > 0 and float(got[DEV][1][6].abs().sum()) == 0


def paged(lens, page, kv, rowlen, window, keep, dtype, seed, before=None):
    """A pool in shuffled pages: pages no query of the step can see (`before[b]`: tokens of row b ahead of this step) are given back
    and hold huge numbers of another request; (cache, block table)."""
    g = torch.Generator().manual_seed(seed)
    need = [-(-n // page) for n in lens]
    pages = sum(need) + 1
    order = torch.randperm(pages, generator=g).tolist()
    cache = torch.randn(pages + 1, kv, page, rowlen, generator=g)
    table = torch.full((len(lens) + 1, max(need) + 1), pages, dtype=torch.int32)
    at = 0
    for b, n in enumerate(need):
        for i in range(n):
            seen_from = max(0, (before[b] if before else 0) - window + 1) if window else 0
            if window and (i + 1) * page <= seen_from and i * page >= keep:
                continue
            table[b, i] = order[at]
            at += 1
    cache[pages] = 0
    return cache.to(dtype), table


MAPS = [(4, 2, 2, 32, 64, 64, 20.0), (20, 1, 1, 48, 80, 64, 0.0), (2, 2, 2, 64, 128, 64, 3.0), (4, 1, 1, 128, 128, 128, 0.0), (24, 2, 2, 16, 48, 16, 5.0),
        (3, 3, 1, 11, 7, 4, 0.0), (3, 1, 2, 9, 13, 16, 2.0), (8, 2, 2, 128, 96, 64, 30.0), (2, 1, 1, 112, 16, 64, 0.5), (2, 1, 2, 40, 24, 64, 0.0), (1, 1, 1, 256, 256, 64, 0.0),
        (34, 1, 2, 8, 8, 64, 9.0), (4, 2, 2, 72, 104, 64, 60.0), (6, 2, 1, 24, 40, 64, 70.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep", [(0, 0), (1, 0), (65, 0), (64, 1), (100, 20), (33, 64), (130, 129), (7, 300)])
@pytest.mark.parametrize("heads,kv,maps,dim,vdim,page,cap", MAPS)
def test_attention_with_maps(K, dtype, window, keep, heads, kv, maps, dim, vdim, page, cap):
    """Rows of one token beside portions of several lengths; scores a few units wide; pages before the window given back."""
    counts, lens = [1, 1, 1, 5, 130, 2, 300], [1, 290, 130, 140, 130, 64, 390]
    before = [n - c for n, c in zip(lens, counts)]
    rowlen, t = maps * dim + vdim, sum(counts)
    cache, table = paged(lens, page, kv, rowlen, window, keep, dtype, 7, before)
    q = rand(t, heads, maps, dim, dtype=dtype, seed=8, scale=2.0)
    wide = rand(t, heads * vdim + 16, dtype=dtype, seed=9, scale=2.0)
    scale, diff = 1.3 / dim ** 0.5, (0.8, 0.4) if maps == 2 else None
    for gated in (True, False) if (window, keep) == (100, 20) else (True,):
        got = {}
        for device, k in (("cpu", REF), (DEV, K)):
            rows = rows_of(counts, list(range(len(counts))), lens, device=device)
            out = torch.full((t, heads, vdim), float("nan"), dtype=dtype if device == DEV else torch.float32, device=device)
            args = (q.to(device), cache.to(device)) if device == DEV else (q.float(), cache.float())
            gate = wide.to(device)[:, 8:8 + heads * vdim] if gated else None
            k.attention_maps(out, *args, table.to(device), rows, scale, cap or None, window, keep if window else 0, diff, 1e-5,
                             gate if gate is None or device == DEV else gate.float())
            got[device] = out
        assert torch.isfinite(got[DEV].float()).all()
        # (two maps: the difference is divided by its own size, which may be small; values spread over about four units then)
        close(got[DEV], got["cpu"], dtype, scale=8.0 if maps == 2 else 2.0)
    if dtype == torch.bfloat16:
        assert K.tcgen05_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("page", [64, 16])
@pytest.mark.parametrize("edge", ["window in", "window out", "first in", "first out", "far", "self"])
def test_one_key_that_takes_all_the_weight(K, dtype, maps, page, edge):
    """One key scores far above all others at an edge of the mask: the output is its value, or does not know it."""
    heads, kv, dim, vdim, window, keep, n = 4, 2, 64, 64, 90, 70, 300
    pos = n - 1
    key = {"window in": pos - window + 1, "window out": pos - window, "first in": keep - 1, "first out": keep, "far": 3, "self": pos}[edge]
    seen = edge in ("window in", "first in", "far", "self")
    for counts in ([1], [2], [150]):
        t, rowlen = sum(counts), maps * dim + vdim
        cache, table = paged([n], page, kv, rowlen, window, keep, dtype, 3, [n - t])
        q = rand(t, heads, maps, dim, dtype=dtype, seed=4)
        special = rand(dim, seed=5).to(dtype)
        q[t - 1, :, 0] = special * 2
        where = int(table[0, key // page])
        if where < cache.shape[0] - 1:
            cache[where, :, key % page, :dim] = special * 2
        else:
            assert not seen
        args = [q.to(DEV), cache.to(DEV), table.to(DEV), rows_of(counts, [0], [n]), 1.0, None, window, keep]
        out = torch.empty(t, heads, vdim, dtype=dtype, device=DEV)
        K.attention_maps(out, *args, (0.6, 0.2) if maps == 2 else None, 1e-5, None)
        want = torch.empty(t, heads, vdim)
        REF.attention_maps(want, q.float(), cache.float(), table, rows_of(counts, [0], [n], device="cpu"), 1.0, None, window, keep,
                           (0.6, 0.2) if maps == 2 else None, 1e-5, None)
        close(out, want, dtype, scale=4.0)
        if maps == 1 and where < cache.shape[0] - 1:
            value = cache[where, :, key % page, dim:].float().repeat_interleave(2, 0)
            near = (out[t - 1].float().cpu() - value).abs().max().item() < 0.05
            assert near == seen


def test_two_maps_that_nearly_cancel(K):
    """λ near 1 and maps of equal keys: what is normed is a small difference of large numbers, which must not be rounded first."""
    heads, kv, dim, vdim, n = 4, 2, 64, 128, 200
    cache, table = paged([n], 64, kv, 2 * dim + vdim, 0, 0, torch.bfloat16, 3)
    cache[..., dim:2 * dim] = cache[..., :dim]
    q = rand(n, heads, 2, dim, dtype=torch.bfloat16, seed=4)
    q[:, :, 1] = (q[:, :, 0].float() * 0.97).to(torch.bfloat16)
    for counts in ([n], [1]):
        qq = q[n - sum(counts):]
        out = torch.empty(sum(counts), heads, vdim, dtype=torch.bfloat16, device=DEV)
        K.attention_maps(out, qq.to(DEV), cache.to(DEV), table.to(DEV), rows_of(counts, [0], [n]), 0.125, 50.0, 0, 0, (0.97, 0.5), 1e-5, None)
        want = torch.empty(sum(counts), heads, vdim)
        REF.attention_maps(want, qq.float(), cache.float(), table, rows_of(counts, [0], [n], device="cpu"), 0.125, 50.0, 0, 0, (0.97, 0.5), 1e-5, None)
        diff = (out.float().cpu() - want).abs()[2 if n == sum(counts) else 0:]
        assert float(diff.pow(2).mean().sqrt()) < 0.08 and float(want.pow(2).mean().sqrt()) > 0.3      # (weights are bfloat16 operands)


# ---------------------------------------------------------------- the model through the replayer
@pytest.fixture(scope="module", params=sorted(CONFIGS))
def model(request, tmp_path_factory):
    folder = make_folder(tmp_path_factory.mktemp("models"), request.param, seed=11)
    config = CONFIGS[request.param]
    prompts = {f"r{i}": random_prompt(config["vocab"], n, 40 + i) for i, n in enumerate((70, 133, 37, 96))}
    return folder, config, prompts, {rid: exact_logits(folder, ids) for rid, ids in prompts.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_then_tail_then_portions(model, dtype):
    folder, config, prompts, want = model
    r = Replayer(str(folder), dtype, 192, device=DEV, page_size=64)
    compare(run(r, [([(rid, ids)], [rid]) for rid, ids in prompts.items()]), want, dtype)
    steps = []
    for rid, ids in prompts.items():                                       # most of it at once, the last 33 one by one
        cut = len(ids) - 33
        steps.append(([(rid, ids[:cut])], []))
        steps += [([(rid, [t])], [rid] if i == 32 else []) for i, t in enumerate(ids[cut:])]
    compare(run(r, steps), want, dtype)
    steps = []
    for rid, ids in prompts.items():                                       # portions down to two tokens, cut inside pages
        parts = portions(ids, [17, 2, 40, 3, 2, 29])
        steps += [([(rid, p)], [rid] if i == len(parts) - 1 else []) for i, p in enumerate(parts)]
    compare(run(r, steps), want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("page_size", [64, 16])
def test_mixed_requests_in_a_small_pool(model, dtype, page_size):
    """Four requests live at once in a pool that holds no more: portions beside single tokens; pages and slots given back
    and taken again; then the same slots and pages for other requests."""
    folder, config, prompts, want = model
    r = Replayer(str(folder), dtype, 448, device=DEV, page_size=page_size)
    got = run(r, mixed_trace(prompts))
    compare(got, want, dtype)
    assert len(got) == sum(len(ids) for ids in prompts.values())
    swapped = {"r0": prompts["r3"], "r3": prompts["r0"]}
    compare(run(r, [([("r0", swapped["r0"][:50]), ("r3", swapped["r3"][:9])], []),
                    ([("r0", swapped["r0"][50:]), ("r3", swapped["r3"][9:])], ["r0", "r3"])]),
            {"r0": want["r3"], "r3": want["r0"]}, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_the_first_tokens(model, dtype):
    folder, config, prompts, want = model
    ids = prompts["r1"]
    r = Replayer(str(folder), dtype, 192, device=DEV, page_size=64)
    steps = [([("r1", [t])], ["r1"] if i == len(ids) - 1 else []) for i, t in enumerate(ids)]      # from the first token on
    compare(run(r, steps), want, dtype)
    steps = [([("r1", ids[:2])], [])] + [([("r1", [t])], ["r1"] if i == len(ids) - 3 else []) for i, t in enumerate(ids[2:])]
    compare(run(r, steps), want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,window,keep", [("diff", 64, 0), ("diff", 65, 0), ("diff", 100, 0), ("par", 33, 64), ("par", 64, 20), ("par", 65, 70), ("par", 2, 1)])
def test_a_key_just_inside_and_just_outside_every_edge(tmp_path, dtype, kind, window, keep):
    """The best key by far lies at an edge's last seen place, then one further: in a prompt, decoded, in portions."""
    reads = 150
    places = [reads - window + 1, reads - window] + ([keep - 1, keep] if kind == "par" else [])
    for key in places:
        config = copy.deepcopy(CONFIGS[kind])
        m = config["layers"][0]["mixer"] if kind == "diff" else config["layers"][0]["mixer"]["left"]
        m["mask"] = {"size": window} if kind == "diff" else {"size": window, "keep_first": keep}
        ids = [3 + t % 80 for t in range(170)]
        ids[reads], ids[key] = 1, 2                                       # two tokens that stand nowhere else
        folder = make_folder(tmp_path / str(key), "edge", config=config, weights=point_at(config, make_weights(config, 3), ids, reads, key))
        want = {"r": exact_logits(folder, ids)}
        r = Replayer(str(folder), dtype, 192, device=DEV, page_size=64)
        for cut in ([170], [140] + [1] * 30, [50, 2, 70, 29, 19]):
            parts = portions(ids, cut)
            compare(run(r, [([("r", p)], ["r"] if i == len(parts) - 1 else []) for i, p in enumerate(parts)]), want, dtype)


def test_a_token_far_back_is_remembered(tmp_path):
    """320 tokens, slow decays: late logits change when token 7, which no window reaches, changes (only the state carries it there),
    and when token 2, a kept one, changes; the engine follows the plain implementation through both, side by side."""
    config = copy.deepcopy(CONFIGS["par"])
    config["layers"][0]["mixer"]["left"]["mask"] = {"size": 20, "keep_first": 4}
    weights = make_weights(config, 3)
    weights["l0.mix.right.A_log"] = torch.tensor([-9.0, -3.0, -7.0, 0.0]).to(torch.bfloat16)
    folder = make_folder(tmp_path, "far", config=config, weights=weights)
    ids = random_prompt(config["vocab"], 320, 5)
    others = {"x": ids}
    for rid, place in (("y", 7), ("z", 2)):
        others[rid] = list(ids)
        others[rid][place] = (ids[place] + 1) % config["vocab"]
    want = {rid: exact_logits(folder, seq) for rid, seq in others.items()}
    r = Replayer(str(folder), "float32", max_tokens=1024)
    steps = [([(rid, seq[:200]) for rid, seq in others.items()], [])] + [([(rid, [seq[i]]) for rid, seq in others.items()], []) for i in range(200, 320)]
    compare(run(r, steps), want, "float32")
    assert all(float((want["x"][300] - want[rid][300]).abs().max()) > 1e-3 for rid in ("y", "z"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wide_layers(tmp_path, dtype):
    """Sizes of the kernels' fast paths together: maps of 64 over values of 128, heads of 128, states of 128 x 64 in parallel, rows of
    512 numbers and more in the norms; 300 tokens whole, the last 40 one by one, and portions that end inside pages."""
    config = _model(512, 331, 1e-6, 0.9, 2.0, [
        _diff(_att(4, 2, 64, 128, 2.0, 130, rot=_rot(1e6, 32), cap=50.0, diff=0.4), 264),
        _par(_att(4, 2, 128, 128, 4.0, 100, 70, _rot(1e6, 64, (8.0, 256, 16.0, 1.0))), _ssm(8, 2, 128, 64, 4, 1), 512),
        _par(_att(2, 1, 64, 64, 4.0, 260, 3, _rot(1e4, 64)), _ssm(16, 1, 64, 64, 4, 2), None)])
    folder = make_folder(tmp_path, "wide", seed=9, config=config)
    ids = random_prompt(config["vocab"], 300, 4)
    want = {"r": exact_logits(folder, ids)}
    r = Replayer(str(folder), dtype, 320, device=DEV, page_size=64)
    for cut in ([300], [260] + [1] * 40, [100, 3, 61, 2, 90, 44]):
        parts = portions(ids, cut)
        compare(run(r, [([("r", p)], ["r"] if i == len(parts) - 1 else []) for i, p in enumerate(parts)]), want, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(model, dtype, graphs):
    from holon_b200.engine import Engine, EngineConfig, SamplingParams
    folder, config, prompts, _ = model
    stored, weights = read_folder(folder)
    engine = Engine(EngineConfig(model=str(folder), dtype=dtype, device=DEV, page_size=16, max_seqs=3, max_model_len=192,
                                 max_step_tokens=64, state_memory=1 << 26, cuda_graphs=graphs))
    asked = [prompts["r0"], prompts["r2"], prompts["r3"][:50], prompts["r1"][:90]]
    with torch.inference_mode():
        got = engine.generate(asked, SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True))
    engine.close()
    gap = 1e-3 if dtype == "float32" else 0.25
    for prompt, tokens in zip(asked, got):
        ids = list(prompt)
        for token in tokens:
            logits = plain.forward(weights, stored, ids)[-1]
            best = int(logits.argmax())
            if token != best:                              # a close call: allowed once, then the sequences part
                assert float(logits[best] - logits[token]) < gap * float(logits.std()), (len(ids), token, best)
                break
            ids.append(token)


def test_generate_on_the_command_line(tmp_path, capsys):
    """`holon-b200 generate` with the engine's own sizing of the cache (activation peaks measured on the largest step)."""
    import json

    from holon_b200 import cli
    folder = make_folder(tmp_path, "a", seed=8)
    config, weights = read_folder(folder)
    assert cli.main(["generate", str(folder), "--prompt-ids", "5,17,3,90,12,7", "--prompt-ids", "9 8 7 6", "--max-tokens", "6",
                     "--dtype", "float32", "--max-model-len", "128", "--max-seqs", "4", "--max-step-tokens", "128", "--ignore-eos",
                     "--memory-fraction", "0.05"]) == 0
    captured = capsys.readouterr()
    lines = [json.loads(line) for line in captured.out.splitlines()]
    assert [o["prompt_ids"] for o in lines] == [[5, 17, 3, 90, 12, 7], [9, 8, 7, 6]]
    for o in lines:
        ids = list(o["prompt_ids"])
        assert len(o["token_ids"]) == 6
        for token in o["token_ids"]:
            logits = plain.forward(weights, config, ids)[-1]
            assert float(logits.max() - logits[token]) <= 1e-3 * float(logits.std()), (len(ids), token)
            ids.append(token)

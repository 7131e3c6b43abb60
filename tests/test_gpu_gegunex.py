"""Gegunex on the GPU. Each new or extended kernel alone against its plain twin (tests/ref_kernels.py) and, where the rule is
short, against the rule written out here in 64-bit, with inputs made so that a fault shows (rows with a large mean, a sink
of the scores' size, one key that takes all the weight just inside or outside a window, row weights far from one, limits
reached on both sides); then the replayer in 32-bit and bfloat16 against the plain implementation (tests/plain_gegunex.py):
whole prompts, prefill against token-by-token decoding, portions down to two tokens, unequal requests mixed in a pool whose
pages and slots are used again, the first tokens, long decoding, sizes that are multiples of nothing, sizes the tensor cores
take; and greedy generation through the engine's scheduler and graphs."""
from __future__ import annotations

import copy
import types

import pytest
import torch

import plain_gegunex as plain
from gegunex_tools import CONFIGS, compare, exact_logits, make_folder, make_weights, point_at, read_folder
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


# ---------------------------------------------------------------- layer norm with what is added first
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,dim", [(7, 64), (3, 72), (5, 1030), (300, 2048), (2, 2048), (4, 33), (300, 5120), (2, 8192), (3, 12288), (3, 11903)])
@pytest.mark.parametrize("weight32", [False, True])
def test_layer_norm(K, dtype, rows, dim, weight32):
    """A row of the stream alone; with a sublayer's row times a factor; with a token's three rows out of a shuffled pile;
    gathered, which leaves the stream as it is. The rows' mean is three times their spread."""
    h, y = rand(rows, dim, seed=1) + 3.0, rand(rows, dim, dtype=dtype, seed=2, scale=2.0)
    pile = rand(3 * rows, dim, dtype=dtype, seed=3)
    place = torch.randperm(3 * rows, generator=torch.Generator().manual_seed(4)).to(torch.int32)
    w = (1 + 0.2 * rand(dim, seed=5)).to(torch.float32 if weight32 else dtype)
    index = torch.tensor([rows - 1, 0, rows - 1], dtype=torch.int32)
    sums = {None: h.to(F64), "row": h.to(F64) + 0.7 * y.to(F64),
            "pairs": h.to(F64) + 0.7 * pile[place.long()].to(F64).view(rows, 3, dim).sum(1)}
    for what, want in sums.items():
        delta = {None: None, "row": y, "pairs": pile}[what]
        args = dict(place=place.to(DEV)) if what == "pairs" else {}
        normed = plain.layer_norm(want, w.to(F64), 1e-5)
        for idx in (None, index):
            hg = h.clone().to(DEV)
            out = torch.empty(rows if idx is None else 3, dim, dtype=dtype, device=DEV)
            K.add_layernorm(out, hg, delta.to(DEV) if delta is not None else None, 0.7, w.to(DEV), 1e-5,
                            idx.to(DEV) if idx is not None else None, **args)
            close(out, normed if idx is None else normed[idx.long()], dtype, scale=2.0)
            if idx is None:
                assert torch.allclose(hg.cpu().to(F64), want, atol=2e-6 * 12)
            else:
                assert torch.equal(hg.cpu(), h), "a gather must write nothing"


def test_layer_norm_of_rows_of_the_engines_dtype(K):
    x = rand(9, 640, dtype=torch.bfloat16, seed=1) + 2.0
    w = (1 + 0.2 * rand(640, seed=2)).to(torch.bfloat16)
    out = torch.empty(9, 640, dtype=torch.bfloat16, device=DEV)
    K.add_layernorm(out, x.to(DEV), None, 1.0, w.to(DEV), 1e-5, None)
    close(out, plain.layer_norm(x.to(F64), w.to(F64), 1e-5), torch.bfloat16, scale=2.0)


@pytest.mark.parametrize("rows,vocab", [(3, 300), (1, 157), (5, 32768)])
def test_soft_limit(K, rows, vocab):
    x = rand(rows, vocab, seed=3, scale=20.0)
    got = x.to(DEV)
    K.softcap(got, 15.0)
    assert torch.allclose(got.cpu().to(F64), 15.0 * torch.tanh(x.to(F64) / 15.0), atol=5e-6)


# ---------------------------------------------------------------- latent attention: a latent for the queries, neighbours, sinks, windows
def turn_table(dims, positions=128, base=300.0, size=1.2):
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    angle = torch.arange(positions, dtype=torch.float32)[:, None] * freq[None]
    return (torch.cat((angle.cos(), angle.sin()), -1) * size).contiguous()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("neighbours", [True, False])
@pytest.mark.parametrize("heads,dim,rot,rank,q_rank", [(3, 20, 12, 40, 22), (4, 64, 32, 64, 96), (1, 16, 64, 512, 1536), (70, 8, 6, 24, 18)])
def test_latent_preparation(K, dtype, neighbours, heads, dim, rot, rank, q_rank):
    """The query latent's norm beside the cache row in one call, the queries' rotation in another."""
    t, page, pages = 9, 4, 5
    first, q = rand(t, q_rank + rank + rot, dtype=dtype, seed=1), rand(t, heads * (dim + rot), dtype=dtype, seed=2)
    positions = torch.tensor([0, 1, 2, 3, 100, 7, 8, 9, 63], dtype=torch.int32)
    widx = torch.tensor([0, 1, 2, 3, 19, 7, -1, 9, 12], dtype=torch.int32)
    table, w, wq = turn_table(rot), (1 + rand(rank, seed=3) * 0.1).to(dtype), (1 + rand(q_rank, seed=4) * 0.1).to(dtype)
    res = []
    for k_, d in ((K, DEV), (REF, "cpu")):
        cq, qa = torch.zeros(t, q_rank, dtype=dtype, device=d), torch.zeros(t, heads, rank + rot, dtype=dtype, device=d)
        cache = torch.zeros(pages, page, rank + rot, dtype=dtype, device=d)
        turn = (positions.to(d), table.to(d), rot)
        k_.latent_prepare(None, first.to(d), heads, dim, rot, rank, q_rank, *turn, w.to(d), 1e-5, cache, widx.to(d),
                          interleaved=neighbours, cq=cq, cq_at=0, cq_weight=wq.to(d))
        k_.latent_prepare(qa, q.to(d), heads, dim, rot, rank, -1, *turn, None, 0.0, None, None, interleaved=neighbours)
        res.append((cq, qa, cache))
    for got, want in zip(*res):
        close(got, want, dtype, scale=4.0)
    cq, qa, cache = res[0]
    close(cq, plain.rms_norm(first[:, :q_rank].to(F64), wq.to(F64), 1e-5), dtype, scale=4.0)
    assert float(cache[1, 2].abs().sum()) == 0.0                            # the skipped token's row (write index -1) stays empty
    if neighbours:                                                          # against the written-out rotation
        cs = table[positions.long()].to(F64)[:, None, :]
        x = q.to(F64).view(t, heads, dim + rot)[:, :, dim:]
        u, v, c, s = x[..., 0::2], x[..., 1::2], cs[..., :rot // 2], cs[..., rot // 2:]
        want = torch.stack((u * c - v * s, v * c + u * s), -1).flatten(-2)
        close(qa[:, :, rank:], want, dtype, scale=4.0)


def paged(lens, page, width, dtype, seed):
    """A cache whose pages are handed out in a scrambled order, and each request's block-table row."""
    need = [-(-n // page) for n in lens]
    pages = sum(need) + 3
    perm = torch.randperm(pages - 1, generator=torch.Generator().manual_seed(seed)).tolist()
    table = torch.full((len(lens), max(need) + 1), pages - 1, dtype=torch.int32)
    at = 0
    for b, n in enumerate(need):
        table[b, :n] = torch.tensor(perm[at:at + n], dtype=torch.int32)
        at += n
    return rand(pages, page, width, dtype=dtype, seed=seed + 1), table


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("splits", [None, 3])
@pytest.mark.parametrize("window", [0, 1, 2, 63, 64, 65, 129])
@pytest.mark.parametrize("heads,rank,rot,page", [(4, 64, 32, 64), (3, 40, 12, 4), (5, 144, 16, 16), (16, 512, 64, 64), (70, 32, 16, 64)])
def test_latent_attention_with_sinks_and_windows(K, dtype, splits, window, heads, rank, rot, page, monkeypatch):
    """Rows of one token (short, at a tile's edge, long) beside portions. For several queries the best key by far lies at
    the window's last seen place, for others one place further back, where it must not be seen; one head's sink dwarfs
    its scores, one head's is far below them."""
    if splits and dtype == torch.float32:
        pytest.skip("the 32-bit kernel does not cut the keys")
    monkeypatch.setattr(K, "latent_split", splits)
    new, lens = [1, 1, 1, 1, 1, 37, 64, 2, 7], [130, 1, 64, 129, 641, 300, 64, 65, 7]      # one-token rows come first
    cache, table = paged(lens, page, rank + rot, dtype, 5)
    t, scale = sum(new), 2.0 / (rank + rot) ** 0.5
    qa = rand(t, heads, rank + rot, dtype=dtype, seed=9)
    sinks = rand(heads, seed=11, scale=1.5) + 1.0
    sinks[0], sinks[-1] = 30.0, -30.0
    host = rows_of(new, list(range(len(new))), lens, device="cpu")
    reach = window or 1 << 20
    marked = []
    for b, (n, length) in enumerate(zip(new, lens)):
        for i, inside in ((n - 1, True), (n - 2, False)):
            if i < 0:
                continue
            pos = length - n + i
            key = pos - (reach - 1 if inside else reach) if window else pos // 3
            if key < 0:
                continue
            row = cache[int(table[b, key // page]), key % page]
            qa[host.host_query_start[b] + i] = (row * (22.0 / float(row.float().pow(2).sum()) / scale)).to(dtype)[None, :]
            marked.append((b, host.host_query_start[b] + i, key, inside or not window))
    out, want = torch.empty(t, heads, rank, dtype=dtype, device=DEV), torch.empty(t, heads, rank, dtype=dtype)
    K.latent_attention(out, qa.to(DEV), cache.to(DEV), table.to(DEV), rows_of(new, list(range(len(new))), lens), scale, rank, window,
                       sinks=sinks.to(DEV))
    REF.latent_attention(want, qa, cache, table, host, scale, rank, window, sinks=sinks)
    close(out, want, dtype, scale=2.0)
    assert float(out[:, 0].abs().max()) < 0.01                              # a sink that takes everything
    for b, q, key, inside in marked:                                        # the last head's sink takes nothing
        value = cache[int(table[b, key // page]), key % page, :rank].float()
        off = float((out[q, heads - 1].float().cpu() - value).abs().max())
        assert (off < 0.1) if inside else (off > 0.1), (b, q, key, inside, off)


# ---------------------------------------------------------------- lightning attention's inputs, a norm over all heads
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim", [(3, 16, 20), (1, 7, 5), (4, 80, 160)])
def test_silu_ahead_of_the_scan(K, dtype, heads, dim, vdim):
    t = 6
    first = rand(t, 2 * heads * dim + 2 * heads * vdim, dtype=dtype, seed=1, scale=2.0)
    qk, v = torch.empty(t, 2, heads, dim, device=DEV), torch.empty(t, heads, vdim, device=DEV)
    positions = torch.arange(t, dtype=torch.int32)
    K.retention_prepare(qk, v, first.to(DEV), positions.to(DEV), None, 0, 1.0, silu=True)
    y, n = plain.silu(first.to(F64)), heads * dim
    assert torch.allclose(qk[:, 0].cpu().to(F64), y[:, :n].view(t, heads, dim), atol=1e-5)
    assert torch.allclose(qk[:, 1].cpu().to(F64), y[:, n:2 * n].view(t, heads, dim), atol=1e-5)
    assert torch.allclose(v.cpu().to(F64), y[:, 2 * n:2 * n + heads * vdim].view(t, heads, vdim), atol=1e-5)
    if dim % 4 == 0:                                                        # silu comes ahead of a rotation
        table = turn_table(dim // 2 * 2 if dim // 2 % 2 == 0 else dim, positions=16)
        K.retention_prepare(qk, v, first.to(DEV), positions.to(DEV), table.to(DEV), table.shape[1], 0.5, silu=True)
        qk_w, v_w = torch.empty(t, 2, heads, dim), torch.empty(t, heads, vdim)
        REF.retention_prepare(qk_w, v_w, first, positions, table, table.shape[1], 0.5, silu=True)
        close(qk, qk_w, torch.float32, scale=2.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("gate", ["sigmoid", "silu"])
@pytest.mark.parametrize("heads,vdim", [(1, 60), (1, 508), (1, 512), (1, 640), (3, 1024), (1, 4096), (1, 11264), (1, 12288), (2, 1030)])
def test_norm_and_gate_of_wide_rows(K, dtype, gate, heads, vdim):
    t, extra = 5, 12
    o, w = rand(t, heads, vdim, seed=1, scale=3.0), 1 + 0.2 * rand(heads * vdim, seed=2)
    wide = rand(t, extra + heads * vdim, dtype=dtype, seed=3)
    out, want = torch.empty(t, heads, vdim, dtype=dtype, device=DEV), torch.empty(t, heads, vdim, dtype=dtype)
    K.head_norm_gate(out, o.to(DEV), w.to(DEV), None, wide.to(DEV)[:, extra:], 1e-5, gate=gate)
    REF.head_norm_gate(want, o, w, None, wide[:, extra:], 1e-5, gate=gate)
    close(out, want, dtype, scale=3.0)
    mul = torch.rand(t, heads, vdim, generator=torch.Generator().manual_seed(5))
    K.head_norm_gate(out, o.to(DEV), None, mul.to(DEV), None, 1e-5)
    REF.head_norm_gate(want, o, None, mul, None, 1e-5)
    close(out, want, dtype, scale=3.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_one_token_rows_move_their_inputs_on(K, dtype, taps):
    """Rows of one token beside portions, in scattered slots, step after step: the carried inputs are the last taps - 1
    inputs of every request whichever kernel moved them on, and slots outside the step keep theirs."""
    heads, kvh, dim, vdim, slots = 4, 2, 12, 20, 6
    c = 2 * kvh * dim + heads * vdim
    conv = rand(c, taps, dtype=dtype, seed=1, scale=0.6)
    dt_bias, rate = rand(heads * dim, seed=3), rand(heads, seed=4)
    cg = rand(slots, taps - 1, c, dtype=dtype, seed=2).to(DEV) if taps > 1 else None
    cw = cg.cpu().clone() if taps > 1 else None
    for step, (counts, where) in enumerate((([1, 1, 5], [4, 0, 2]), ([1, 1], [2, 4]), ([1, 2, 1], [5, 0, 2]), ([1], [0]))):
        t = sum(counts)
        first, low2 = rand(t, c + heads, dtype=dtype, seed=20 + step), rand(t, heads * (dim + vdim), seed=30 + step)
        outs = []
        for k_, d, state in ((K, DEV, cg), (REF, "cpu", cw)):
            e = lambda *s: torch.empty(*s, device=d)                        # noqa: E731
            bufs = (e(t, 2, kvh, dim), e(t, heads, vdim), e(t, heads), e(t, heads, dim), e(t, heads * vdim))
            rows = rows_of(counts, where, device=d)
            k_.delta_prepare(*bufs, first.to(d), conv.to(d), state, low2.to(d), dt_bias.to(d), rate.to(d), rows, dim ** -0.5, 1e-6,
                             carry=True)
            k_.conv_carry(state, first.to(d), c, taps, rows, least=2)
            outs.append(bufs)
        for got, want in zip(*outs):
            close(got, want, torch.float32, scale=3.0)
        if taps > 1:
            assert torch.equal(cg.cpu(), cw), step


# ---------------------------------------------------------------- experts: sigmoid scores, weights ahead of the limits
@pytest.mark.parametrize("experts,top,tokens", [(16, 4, 8), (5, 5, 64), (1, 1, 3), (300, 8, 33), (9, 2, 300), (1100, 3, 20), (12, 1, 700)])
@pytest.mark.parametrize("grouped", [False, True])
def test_sigmoid_scores(K, experts, top, tokens, grouped):
    """Few tokens take one launch, many (or more than 1,024 experts) the separate kernels; with a correction, the warp that
    chooses under one. Every row carries its pair's weight."""
    z = rand(tokens, experts, seed=4, scale=2.0)
    corr = rand(experts, seed=5, scale=0.2) if grouped else None
    kw = dict(scores="sigmoid") | (dict(correction=corr, tiny=1e-20) if grouped else {})
    for renorm in (False, True):
        chosen, weight = torch.empty(tokens, top, dtype=torch.int32, device=DEV), torch.empty(tokens, top, device=DEV)
        counts = torch.full((2 * experts + 3,), -7, dtype=torch.int32, device=DEV)
        place, token_of = (torch.empty(tokens * top, dtype=torch.int32, device=DEV) for _ in range(2))
        row_weight = torch.empty(tokens * top, device=DEV)
        K.route_rows(chosen, weight, counts, place, token_of, z.to(DEV), experts, 0.6, renorm, row_weight=row_weight,
                     **{k: v.to(DEV) if torch.is_tensor(v) else v for k, v in kw.items()})
        s = torch.sigmoid(z.to(F64))
        order = torch.argsort(-(s + (corr.to(F64) if grouped else 0.0)), dim=-1, stable=True)[:, :top]
        w = torch.gather(s, 1, order)
        w = 0.6 * (w / w.sum(-1, keepdim=True) if renorm else w)
        assert torch.equal(chosen.cpu().long(), order)
        assert torch.allclose(weight.cpu().to(F64), w, rtol=1e-5)
        assert torch.equal(row_weight.cpu()[place.cpu().long()], weight.cpu().reshape(-1))
        assert torch.equal(counts.cpu()[:experts].long(), torch.bincount(order.reshape(-1), minlength=experts))


@pytest.mark.parametrize("dtype,mode", [(torch.float32, "fast"), (torch.bfloat16, "fast"), (torch.bfloat16, "tcgen05"), (torch.bfloat16, "mma"),
                                        (torch.bfloat16, "generic")])
@pytest.mark.parametrize("experts,top,tokens,hidden,inter", [(6, 2, 50, 72, 40), (16, 4, 3, 64, 96), (3, 3, 130, 40, 24), (40, 1, 9, 32, 8),
                                                             (5, 2, 400, 328, 136), (4, 2, 900, 264, 200), (3, 1, 70, 100, 52), (2, 2, 1, 2048, 384), (2, 1, 3, 3072, 8), (2, 1, 3, 8, 3072)])
def test_clamped_experts(K, dtype, mode, experts, top, tokens, hidden, inter, monkeypatch):
    """From router logits to the sum, against the twin and the rule written out: experts without rows, partial tiles, sizes
    that are multiples of 4 only; gates and ups on both sides of the limit; weights from near 0 to near 1."""
    monkeypatch.setattr(K, "expert_products", mode)
    limit, alpha = 0.9, 1.702
    z = rand(tokens, experts, seed=1, scale=2.0)
    if experts > 4:
        z[:, 1] = -50.0                                                      # an expert nobody chooses
    x = rand(tokens, hidden, dtype=dtype, seed=2)
    up, down = rand(experts, 2 * inter, hidden, dtype=dtype, seed=3, scale=1.5 * hidden ** -0.5), rand(experts, hidden, inter, dtype=dtype, seed=4, scale=inter ** -0.5)
    res = []
    for k_, d in ((K, DEV), (REF, "cpu")):
        chosen, weight = torch.empty(tokens, top, dtype=torch.int32, device=d), torch.empty(tokens, top, device=d)
        counts = torch.zeros(2 * experts + 3, dtype=torch.int32, device=d)
        place, token_of = (torch.empty(tokens * top, dtype=torch.int32, device=d) for _ in range(2))
        row_weight = torch.empty(tokens * top, device=d)
        k_.route_rows(chosen, weight, counts, place, token_of, z.to(d), experts, 1.0, False, scores="sigmoid", row_weight=row_weight)
        starts = counts[experts:2 * experts + 1]
        act, y = torch.empty(tokens * top, inter, dtype=dtype, device=d), torch.empty(tokens * top, hidden, dtype=dtype, device=d)
        k_.expert_glu(act, x.to(d), token_of, up.to(d), starts, limit, alpha, row_weight)
        k_.expert_linear(y, act, None, down.to(d), starts, 0)
        out = torch.empty(tokens, hidden, dtype=dtype, device=d)
        k_.expert_combine(out, y, place, None, None, None, 0)
        order = place.cpu().long()
        res.append((act.cpu()[order], out))
    close(res[0][0], res[1][0], dtype, scale=2.0)
    close(res[0][1], res[1][1], dtype, scale=4.0)
    weights = {f"e{e}.{n}": t for e in range(experts) for n, t in (("gate", up[e, :inter]), ("up", up[e, inter:]), ("down", down[e]))}
    want = torch.zeros(tokens, hidden, dtype=F64)
    for t in range(min(tokens, 60)):
        for e, share in plain.choose(z[t].to(F64), top):
            want[t] += plain.clamped_unit(share * x[t].to(F64), weights, f"e{e}.", limit)
    close(res[0][1][:60], want[:60], dtype, scale=4.0)
    if mode == "tcgen05":
        assert K.tcgen05_status() == 0


def test_clamped_unit_without_row_weights(K):
    x, w = rand(5, 64, dtype=torch.bfloat16, seed=1), rand(2, 48, 64, dtype=torch.bfloat16, seed=2, scale=0.2)
    starts = torch.tensor([0, 2, 5], dtype=torch.int32)
    for tile in (0, 16):
        K.expert_tile_rows = tile
        try:
            out, want = torch.empty(5, 24, dtype=torch.bfloat16, device=DEV), torch.empty(5, 24, dtype=torch.bfloat16)
            K.expert_glu(out, x.to(DEV), None, w.to(DEV), starts.to(DEV), 0.8, 1.702, None)
        finally:
            K.expert_tile_rows = 0
        REF.expert_glu(want, x, None, w, starts, 0.8, 1.702, None)
        close(out, want, torch.bfloat16)


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
@pytest.mark.parametrize("window", [1, 64, 65, 100])
def test_a_key_just_inside_and_just_outside_the_window(tmp_path, dtype, window):
    """The best key by far lies at the window's last seen place (then one further back): in a prompt, decoded, in portions."""
    reads = 150
    for distance in (window - 1, window):
        if not distance:
            continue
        config = copy.deepcopy(CONFIGS["lat"])
        config["layers"][0]["mixer"]["mask"]["size"] = window
        ids = [3 + t % 80 for t in range(170)]
        ids[reads], ids[reads - distance] = 1, 2                          # two tokens that stand nowhere else
        weights = point_at(config, make_weights(config, 3), 0, ids, reads, reads - distance, 12.0)
        folder = make_folder(tmp_path / str(distance), "edge", config=config, weights=weights)
        want = {"r": exact_logits(folder, ids)}
        r = Replayer(str(folder), dtype, 192, device=DEV, page_size=64)
        for cut in ([170], [140] + [1] * 30, [50, 2, 70, 29, 19]):
            parts = portions(ids, cut)
            compare(run(r, [([("r", p)], ["r"] if i == len(parts) - 1 else []) for i, p in enumerate(parts)]), want, dtype)


def test_a_token_far_back_is_remembered(tmp_path):
    """Matrix-state layers alone, 320 tokens, slow decays: late logits change when token 7 changes (only the state can carry
    it there), and the engine follows the plain implementation through that change, with both requests side by side."""
    config = copy.deepcopy(CONFIGS["lin"])
    config["layers"][0]["mixer"]["decay"] = [0.6, 0.97, 0.999]
    config["layers"] += copy.deepcopy(CONFIGS["delta"]["layers"])
    folder = make_folder(tmp_path, "far", seed=3, config=config)
    ids = random_prompt(config["vocab"], 320, 5)
    other = list(ids)
    other[7] = (ids[7] + 1) % config["vocab"]
    want = {"x": exact_logits(folder, ids), "y": exact_logits(folder, other)}
    r = Replayer(str(folder), "float32", max_tokens=768)
    steps = [([("x", ids[:200]), ("y", other[:200])], [])] + [([("x", [a]), ("y", [b])], []) for a, b in zip(ids[200:], other[200:])]
    compare(run(r, steps), want, "float32")
    assert float((want["x"][300] - want["y"][300]).abs().max()) > 1e-3        # the changed token matters to late rows


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wide_layers(tmp_path, dtype):
    """Sizes of the kernels' fast paths together: a latent of 512 with a rotated part of 64, matrix states of 128 x 128,
    experts whose prompt rows run on tcgen05; 300 tokens whole, the last 40 one by one, and portions that end inside pages."""
    from gegunex_tools import _delta, _lat, _layer, _lin, _model, _moe
    config = _model(256, 331, 1e-6, 0.9, 25.0, [
        _layer("latent_attention", _lat(4, 128, 64, 128, 192, 512, 130, 3.0, 1e6, (8.0, 256, 16.0, 1.0)), _moe(3, 1, 136, 2.0)),
        _layer("channel_delta", _delta(4, 2, 128, 128, 4, 20, 12), _moe(2, 2, 64, 1.0)),
        _layer("lightning", _lin(2, 128, 128), None)])
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

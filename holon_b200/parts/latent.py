"""Latent attention over a paged cache of one row per token.

Per token the layer keeps only c (the RMS-normed first `rank` outputs of the down-projection) and k_r (its last
`rot_dim` outputs, rotated by the token's position), which all heads share. Head h has queries q_h = [q_h^u (dim
unrotated) | q_h^r (rot_dim, rotated)], keys k_{h,j} = [W_uk,h c_j | k_r,j] and values v_{h,j} = W_uv,h c_j, and

    score_h(i, j) = (q_h^u(i) · W_uk,h c_j + q_h^r(i) · k_r,j) · scale,   j ≤ i,   softmax over j,
    out_h(i) = W_uv,h Σ_j p_h(i, j) c_j,   then · sigmoid(W_g x) element by element, then W_o.

Because W_uk,h and W_uv,h act on the cached row only, they are applied on the query's side: a_h(i) = W_uk,hᵀ q_h^u(i)
(`rank` numbers) makes q_h^u · W_uk,h c_j = a_h · c_j, so every head attends over the same rows [c_j | k_r,j] with
the query [a_h | q_h^r], the attention's value is c_j itself, and W_uv,h is applied once to the weighted sum. Keys and
values per head are never made; that holds for prompts and for decoding alike.

A layer without a down-projection of its own (`own_latent=False`) reads the cache entry another layer fills (the
run order says which) with its own W_uk, W_uv, queries, gate and output product.

The first products (q, gate, down-projection) are one merged product; the rotation table is the position part's.

Options that other designs use: `q_rank` (queries come from a latent of their own: q = W_uq RMSnorm(W_dq x), stored as dq,
dq.norm, uq; W_dq takes q's place in the merged product), `gate=False` (no output gate, no g), `sink` (one learned number per
head, stored as `sink`: exp(sink) stands in the softmax's denominator, without key or value and without the score scale),
`window` W > 0 (a query at position p sees only keys with p − j < W).
"""
from __future__ import annotations

import torch

from ..config.spec import PartRef
from .base import BuildContext, PagedLatent, Part
from .linear import Linear


class LatentAttention(Part):
    def __init__(self, ctx: BuildContext, *, heads: int, dim: int, rot_dim: int, vdim: int, rank: int, scale: float,
                 hidden: int, norm: PartRef, position: PartRef | None, own_latent: bool = True, window: int = 0,
                 q_rank: int | None = None, gate: bool = True, sink: bool = False, layer: int = 0) -> None:
        super().__init__()
        self.ctx, self.heads, self.dim, self.rot_dim, self.vdim, self.rank = ctx, heads, dim, rot_dim, vdim, rank
        self.scale, self.own_latent, self.window = float(scale), bool(own_latent), int(window)
        self.q_rank, self.gate = q_rank, bool(gate)
        self.n_q = heads * (dim + rot_dim) if q_rank is None else q_rank          # columns of the first product ahead of the gate's
        pieces = {"q": self.n_q} if q_rank is None else {"dq": q_rank}
        if gate:
            pieces["g"] = heads * vdim
        if own_latent:
            pieces["dkv"] = rank + rot_dim
        self.first = self.add_child("first", Linear(ctx, "weight", hidden, pieces))
        self.q_norm = self.uq = None
        if q_rank is not None:
            self.q_norm = self.add_child("q_norm", ctx.part(norm, dim=q_rank))
            self.uq = self.add_child("up_q", Linear(ctx, "weight", q_rank, {"uq": heads * (dim + rot_dim)}))
        self.sink = self.add_param("sink", (heads,), "coef") if sink else None
        self.uk = self.add_param("uk", (heads * dim, rank), "matrix")
        self.uv = self.add_param("uv", (heads * vdim, rank), "matrix")
        self.out = self.add_child("out", Linear(ctx, "weight", heads * vdim, {"o": hidden}))
        self.latent_norm = self.add_child("latent_norm", ctx.part(norm, dim=rank)) if own_latent else None
        self.position = self.add_child("position", ctx.part(position, head_dim=rot_dim)) if position and rot_dim else None
        self.uk_t = None                    # [heads, rank, dim]: W_uk per head, transposed (made in finalize)

    def loadables(self, prefix: str = ""):
        """Stored names: q (or dq, dq.norm, uq), g, dkv, dkv.norm, uk, uv, sink, o."""
        rename = {prefix + "latent_norm.weight": prefix + "dkv.norm", prefix + "q_norm.weight": prefix + "dq.norm"}
        for name, p, rows in super().loadables(prefix):
            for child in ("first.", "up_q.", "out."):
                if name.startswith(prefix + child):
                    name = prefix + name[len(prefix + child):]
            yield rename.get(name, name), p, rows

    def finalize(self) -> None:
        super().finalize()
        if self.uk.tensor is not None:
            self.uk_t = self.uk.tensor.view(self.heads, self.dim, self.rank).transpose(1, 2).contiguous()

    def cache(self) -> PagedLatent:
        return PagedLatent(self.rank, self.rot_dim, self.window)

    def slot_states(self):
        return ()

    @property
    def plan_group(self):
        return "latent", self.heads, self.rank, self.rot_dim, self.window

    def capture_plan(self, step, max_model_len: int):
        plan = getattr(self.ctx.kernels, "attention_capture_plan", None)
        return plan(step.rows, max_model_len) if plan is not None else None

    def forward(self, x: torch.Tensor, step, cache) -> torch.Tensor:
        t, k, ctx = x.shape[0], self.ctx.kernels, self.ctx
        heads, dim, rot, rank, vdim = self.heads, self.dim, self.rot_dim, self.rank, self.vdim
        fills = cache.fills and self.own_latent
        first = self.first.forward(x)                                   # [t, q or dq | g | dkv]
        n_q, n_g = self.n_q, heads * vdim if self.gate else 0
        pos = self.position
        qa = ctx.empty(t, heads, rank + rot)                             # the folded queries [a_h | q_h^r]
        turn = (step.positions, pos.table if pos else None, pos.rotary_dim if pos else 0)
        neighbours = {"interleaved": True} if pos is not None and pos.interleaved else {}
        row = (self.latent_norm.weight.tensor, self.latent_norm.eps, cache.kv, cache.group.write_index) if fills \
            else (None, self.q_norm.eps if self.q_norm else 0.0, None, None)
        at = n_q + n_g if fills else -1
        if self.uq is None:
            q = first
            k.latent_prepare(qa, first, heads, dim, rot, rank, at, *turn, *row, **neighbours)
        else:                                                            # cache row and query latent, then the queries' rotation
            cq = ctx.empty(t, self.q_rank)
            k.latent_prepare(None, first, heads, dim, rot, rank, at, *turn, *row, cq=cq, cq_at=0,
                             cq_weight=self.q_norm.weight.tensor, **neighbours)
            q = self.uq.forward(cq)
            k.latent_prepare(qa, q, heads, dim, rot, rank, -1, *turn, None, 0.0, None, None, **neighbours)
        q_u = q[:, :heads * (dim + rot)].view(t, heads, dim + rot)[:, :, :dim]
        k.linear_heads(qa[:, :, :rank], q_u, self.uk_t)                   # a_h = W_uk,hᵀ q_h^u
        mix = ctx.empty(t, heads, rank)
        sinks = {"sinks": self.sink.tensor} if self.sink is not None else {}
        k.latent_attention(mix, qa, cache.kv, cache.group.block_table, step.rows, self.scale, rank, self.window, **sinks)
        o = ctx.empty(t, heads, vdim)
        k.linear_heads(o, mix, self.uv.tensor.view(heads, vdim, rank))    # W_uv,h on the weighted sum of latents
        o = o.view(t, heads * vdim)
        if self.gate:
            k.sigmoid_gate(o, first[:, n_q:n_q + n_g])
        return self.out.forward(o)

"""Latent attention: keys and values are made from one small vector per token, and only that vector is cached.

With h the mixer's input: q = Wq h (heads x dim); c = rms_norm(Wdkv h) (size rank, a plain weight, eps inside the
root) is the token's latent; per head k = Wuk c (dim), v = Wuv c (vdim); score = (q . k) * scale; position i sees
every j <= i; softmax; the concatenated heads are projected by Wo.  There are no positions.  A layer may have no
Wdkv of its own and attend over the latents another layer cached (a place of the schedule that reads an earlier
place's cache), with its own Wuk, Wuv, queries and output.

Since k and v are linear in c, the products with Wuk and Wuv move to the other side of the attention:
  q . (Wuk_h c) = (Wuk_h^T q_h) . c          and          sum_j p_j Wuv_h c_j = Wuv_h (sum_j p_j c_j),
so the attention is multi-query attention over the cached latents themselves (one key/value head of size rank whose
values are its keys), with queries Wuk_h^T Wq_h h and output Wo_h Wuv_h o_h.  Both pairs of matrices are multiplied
once when the weights are loaded (in float64, then rounded to the engine dtype), so a step runs two products, one
small kernel (queries to the engine dtype, the latent's norm and its append to the pages) and the library's
grouped-query attention with head size rank.  Cached per token: rank numbers, whatever the heads.

`rotary_latent_attention` further down is the form with a rotated key part beside the latent and an output gate.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .attention import _check_kernel_limits, attend_paged, stored_head_size
from .base import KVSpec, Mixer, PartSpec, register_part, shared_part
from .linear import Linear


class LatentAttention(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, dim: int, vdim: int, rank: int, scale: float, eps: float,
                 own_latent: bool = True, dtype: torch.dtype = torch.bfloat16,
                 device: torch.device = torch.device("cuda")):
        self.hidden_size, self.nh, self.dim, self.vdim, self.rank = (int(hidden_size), int(num_heads), int(dim),
                                                                      int(vdim), int(rank))
        self.scale, self.eps, self.own_latent = float(scale), float(eps), bool(own_latent)
        self.dtype, self.device = dtype, device
        # the attention runs with head size rank and one kv head (a rank that the bfloat16 kernels do not take is
        # stored as the next size they take: zero rows in the queries' matrix, zero columns in the output's)
        self.rank_stored = stored_head_size(self.rank, dtype)
        _check_kernel_limits(self.nh, 1, self.rank_stored, dtype)
        self.q_width = self.nh * self.rank_stored
        # rows: the queries in latent space, then (own latent) the latent's projection
        self.proj = Linear(hidden_size, self.q_width + (self.rank if self.own_latent else 0), dtype, device,
                           name="q_dkv" if self.own_latent else "q", pad_width=True)
        self.q_only: Optional[Linear] = None
        self.o = Linear(self.q_width, hidden_size, dtype, device, name="o", pad_width=True)
        self.norm_weight: Optional[torch.Tensor] = None

    def cache_spec(self) -> Optional[KVSpec]:
        return KVSpec(1, self.rank_stored, values_are_keys=True) if self.own_latent else None

    def weight_shapes(self):
        shapes = {"q": ((self.nh * self.dim, self.hidden_size), "normal"),
                  "uk": ((self.nh * self.dim, self.rank), "normal"), "uv": ((self.nh * self.vdim, self.rank), "normal"),
                  "o": ((self.hidden_size, self.nh * self.vdim), "normal")}
        if self.own_latent:
            shapes.update(dkv=((self.rank, self.hidden_size), "normal"), dkv_norm=((self.rank,), "ones"))
        return shapes

    def load(self, q, uk, uv, o, dkv=None, dkv_norm=None) -> None:
        H, d, e, r, W = self.nh, self.dim, self.vdim, self.rank, self.hidden_size
        for name, t, shape in (("q", q, (H * d, W)), ("uk", uk, (H * d, r)), ("uv", uv, (H * e, r)), ("o", o, (W, H * e))):
            if tuple(t.shape) != shape:
                raise ValueError(f"weight '{name}' of shape {tuple(t.shape)} does not fit {shape}")
        f64 = lambda t: t.to(device=self.device, dtype=torch.float64)      # noqa: E731
        # queries into latent space: rows [head][rank] = Wuk_h^T Wq_h
        rp = self.rank_stored
        q_latent = torch.zeros((H, rp, W), dtype=torch.float64, device=self.device)
        q_latent[:, :r] = torch.einsum("hdr,hdw->hrw", f64(uk).view(H, d, r), f64(q).view(H, d, W))
        q_latent = q_latent.reshape(H * rp, W)
        # the output from latent space: columns [head][rank] = Wo_h Wuv_h
        o_latent = torch.zeros((W, H, rp), dtype=torch.float64, device=self.device)
        o_latent[:, :, :r] = torch.einsum("whe,her->whr", f64(o).view(W, H, e), f64(uv).view(H, e, r))
        o_latent = o_latent.reshape(W, H * rp)
        if self.own_latent:
            if dkv is None or dkv_norm is None or tuple(dkv_norm.shape) != (r,):
                raise ValueError("a latent attention layer with a latent of its own needs 'dkv' and 'dkv_norm'")
            self.proj.load([q_latent, f64(dkv)])
            self.norm_weight = dkv_norm.to(device=self.device, dtype=torch.float32).contiguous()
        else:
            self.proj.load([q_latent])
        self.q_only = self.proj.first_rows(self.q_width)
        self.o.load([o_latent])

    def _linear(self, writes_cache: bool) -> Linear:
        if writes_cache and not self.own_latent:
            raise ValueError("this latent attention layer has no latent of its own: it must read another place's cache")
        return self.proj if writes_cache else self.q_only

    def scratch_to_clear(self, ctx, tokens: int, writes_cache: bool = True) -> Optional[torch.Tensor]:
        """The projections' float32 buffer, if this step's product adds slices of K into it (decode-sized steps):
        the launch before this mixer clears it in passing."""
        lin = self._linear(writes_cache)
        if lin is None or not lin.meets_by_adds(tokens, torch.float32):
            return None
        buf = ctx.workspace.get("latent_proj", (tokens, lin.out_features), torch.float32)
        return buf if buf.numel() % 4 == 0 else None

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx, cache_view, writes_cache: bool = True,
                scratch_cleared: bool = False) -> None:
        T = x.shape[0]
        ws = ctx.workspace
        group = cache_view.group
        lin = self._linear(writes_cache)
        proj = ws.get("latent_proj", (T, lin.out_features), torch.float32)
        lin.forward(x, proj, y_is_zero=scratch_cleared)
        q = ws.get("latent_q", (T, self.q_width), self.dtype)
        ops.latent_prep(proj, self.q_width, self.rank, self.norm_weight, self.eps, q, group.dest_rows, cache_view.k,
                        write_c=writes_cache, stored_rank=self.rank_stored)
        attn = ws.get("latent_attn", (T, self.q_width), self.dtype)
        attend_paged(q, cache_view.k, cache_view.k, attn, ctx, group, self.nh, 1, self.rank_stored, 0, self.scale)
        self.o.forward_add(attn, residual)


register_part("mixer", "latent_attention", LatentAttention)


# Constants of the estimate in `RotaryLatentAttention._as_heads` (operations per microsecond): they rank the two ways
# of a prompt step, they forecast no time.
_PRODUCT_FLOPS_PER_US = 1.0e9      # the product that makes keys and values, tcgen05
_HEADS_FLOPS_PER_US = 5.0e8        # attention over them, tcgen05
_LATENT_FLOPS_PER_US = 1.5e8       # attention over the rows themselves, mma.sync
_HEADS_FIXED_US = 12.0             # two more launches
_HEADS_MAX_BYTES = 6 << 30         # of the matrix of keys and values of one step
_LATENT_MAX_BYTES = 2 << 30        # of the queries in the latents' space of one launch


class RotaryLatentAttention(Mixer):
    """Latent attention with a rotated part and an output gate.

    With h the mixer's input: q = Wq h, per head d unrotated then r rotated numbers; Wdkv h has n + r rows, the first n
    divided by their root mean square (eps inside the root) and multiplied by a weight are the token's latent c, the
    last r are one rotated key part p that all heads share.  Rotation turns the pair (i, i + r/2) of the queries' rotated
    numbers and of p by the position's angle.  Per head k = [Wuk c | p], v = Wuv c, score = (q . k) * scale, position i
    sees every j <= i, softmax.  The concatenated heads are multiplied by sigmoid(Wg h) (`gate`) and projected by Wo.
    The cache holds [c | p] per token, whatever the heads; a layer without a latent of its own (`own_latent` False)
    reads the rows that an earlier place cached, with its own Wuk, Wuv, queries, gate and output.

    Options: `q_rank` m: the queries have a latent of their own, q = Wuq (rms_norm(Wdq h)) with a weight of size m
    (one launch norms it, finishes the token's row and clears what the product behind it adds into).  `gate` "head": one
    number per head, sigmoid(Wg h)_h times the head's output; the attention over heads applies it to its sums and the values'
    kernel to its own.  `pairs` "neighbours": the rotation turns the pair (2 i, 2 i + 1); the rows of the matrices that make
    the rotated numbers, of the queries and of p alike, are put in the order of the halves when they are loaded, which
    leaves every score as it is.

    Two ways through a step of the bfloat16 engine, picked by an estimate of the time:
    - in the latents' space (single tokens, short portions behind long histories): the query passes Wuk on its side,
      q' = [Wuk^T q | turned q], a cached row is the key of all heads and its first n numbers their value
      (`ops.latent_attention`), and the weighted sum of latents passes Wuv afterwards.  Three small launches around the
      products: queries and the token's row, the attention, values with the gate (which also joins the key splits).
    - as heads (prompts): one product over the rows of the step's sequences makes every head's keys and values (the
      rotated part rides through it by rows of an identity: a row [c | p] times [Wuk_h 0; 0 I] is the head's key), then
      attention with a key head per query head on the tcgen05 tensor cores.
    The float32 engine always works in the latents' space."""

    prompt_way: Optional[str] = None         # "heads" or "latents": every prompt step goes that way (for measurements)

    def __init__(self, hidden_size: int, num_heads: int, dim: int, rot_dim: int, vdim: int, rank: int, scale: float,
                 eps: float, position: Optional[PartSpec] = None, gate=True, own_latent: bool = True,
                 q_rank: Optional[int] = None, pairs: str = "halves",
                 dtype: torch.dtype = torch.bfloat16, device: torch.device = torch.device("cuda")):
        self.hidden_size, self.nh, self.dim, self.rot, self.vdim, self.rank = (
            int(hidden_size), int(num_heads), int(dim), int(rot_dim), int(vdim), int(rank))
        if gate not in (True, False, "head") or pairs not in ("halves", "neighbours"):
            raise ValueError(f"a gate is True, False or 'head', pairs are 'halves' or 'neighbours', got {gate!r}, {pairs!r}")
        self.q_rank = None if q_rank is None else int(q_rank)
        self.head_gate, self.neighbours = gate == "head", pairs == "neighbours"
        if self.rot % 2:
            raise ValueError(f"{self.rot} rotated numbers do not form pairs")
        self.scale, self.eps, self.gate, self.own_latent = float(scale), float(eps), gate is not False, bool(own_latent)
        self.dtype, self.device = dtype, device
        self.row = stored_head_size(self.rank + self.rot, dtype)          # numbers a cached row is stored with
        if self.row > ops.LATENT_MAX_ROW or (dtype == torch.bfloat16
                                             and not ops.latent_attention_supported(self.row, self.rank)):
            raise ValueError(f"cached rows of {self.rank} + {self.rot} numbers are not supported (at most "
                             f"{ops.LATENT_MAX_ROW})")
        self.position = shared_part("position", position, dtype, device) if position is not None else None
        # columns of the stacked projection: queries (or their latent), gate, then the row (a view of the first columns
        # serves places that read another place's rows)
        self.q_width, self.o_width = self.nh * (self.dim + self.rot), self.nh * self.vdim
        self.gate_width = (self.nh if self.head_gate else self.o_width) if self.gate else 0
        self.gate_col = self.q_width if self.q_rank is None else self.q_rank
        self.row_col = self.gate_col + self.gate_width
        self.uq: Optional[Linear] = None
        self.q_norm_weight: Optional[torch.Tensor] = None
        if self.q_rank is not None:
            self.uq = Linear(self.q_rank, self.q_width, dtype, device, name="uq", pad_width=True)
        self.proj = Linear(hidden_size, self.row_col + (self.rank + self.rot if self.own_latent else 0), dtype, device,
                           name="q_g_dkv" if self.own_latent else "q_g", pad_width=True)
        self.q_only: Optional[Linear] = None
        # heads as they are stored for the output product (and, in bfloat16, for attention as heads)
        self.v_stored = stored_head_size(self.vdim, dtype)
        self.k_stored = max(stored_head_size(self.dim + self.rot, dtype), self.v_stored)
        self.o = Linear(self.nh * self.v_stored, hidden_size, dtype, device, name="o", pad_width=True)
        self.heads_width = self.nh * (self.k_stored + self.v_stored)
        self.to_heads: Optional[Linear] = None
        if dtype == torch.bfloat16 and ops.attention_tc_supported(self.nh, self.nh, self.k_stored):
            self.to_heads = Linear(self.row, self.heads_width, dtype, device, name="latent_to_heads")
        self.norm_weight = self.uk = self.uv = None

    def cache_spec(self) -> Optional[KVSpec]:
        return KVSpec(1, self.row, values_are_keys=True) if self.own_latent else None

    def limit_positions(self, n: int) -> None:
        limit = getattr(self.position, "limit_positions", None)
        if limit is not None:
            limit(n)

    def weight_shapes(self):
        H, W, n = self.nh, self.hidden_size, self.rank
        shapes = {"uk": ((H * self.dim, n), "normal"), "uv": ((H * self.vdim, n), "normal"),
                  "o": ((W, self.o_width), "normal")}
        if self.q_rank is None:
            shapes["q"] = ((self.q_width, W), "normal")
        else:
            m = self.q_rank
            shapes.update(dq=((m, W), "normal"), dq_norm=((m,), "ones"), uq=((self.q_width, m), "normal"))
        if self.gate:
            shapes["g"] = ((self.gate_width, W), "normal")
        if self.own_latent:
            shapes.update(dkv=((n + self.rot, W), "normal"), dkv_norm=((n,), "ones"))
        return shapes

    def _halves(self, w: torch.Tensor, heads: int, before: int) -> torch.Tensor:
        """Rows of `heads` groups of before + r: with pairs of neighbours, the last r of a group as the even ones, then the
        odd ones."""
        if not self.neighbours or self.rot == 0:
            return w
        group = before + self.rot
        order = list(range(before)) + [before + i for s in (0, 1) for i in range(s, self.rot, 2)]
        return w.reshape(heads, group, w.shape[1])[:, order].reshape(heads * group, w.shape[1])

    def load(self, uk, uv, o, q=None, dq=None, dq_norm=None, uq=None, g=None, dkv=None, dkv_norm=None) -> None:
        H, d, r, e, n, W = self.nh, self.dim, self.rot, self.vdim, self.rank, self.hidden_size
        for name, t, shape in (("uk", uk, (H * d, n)), ("uv", uv, (H * e, n)), ("o", o, (W, H * e))):
            if tuple(t.shape) != shape:
                raise ValueError(f"weight '{name}' of shape {tuple(t.shape)} does not fit {shape}")
        if self.own_latent and (dkv is None or dkv_norm is None or tuple(dkv_norm.shape) != (n,)):
            raise ValueError("a latent attention layer with a latent of its own needs 'dkv' and 'dkv_norm'")
        if self.q_rank is not None:
            if tuple(dq_norm.shape) != (self.q_rank,):
                raise ValueError(f"weight 'dq_norm' of shape {tuple(dq_norm.shape)} does not fit ({self.q_rank},)")
            self.q_norm_weight = dq_norm.to(device=self.device, dtype=torch.float32).contiguous()
            self.uq.load([self._halves(uq, H, d)])
        self.proj.load([self._halves(q, H, d) if self.q_rank is None else dq] + ([g] if self.gate else [])
                       + ([self._halves(dkv, 1, n)] if self.own_latent else []))
        self.q_only = self.proj.first_rows(self.row_col)
        if self.own_latent:
            self.norm_weight = dkv_norm.to(device=self.device, dtype=torch.float32).contiguous()
        self.uk = uk.to(device=self.device, dtype=self.dtype).contiguous()
        self.uv = uv.to(device=self.device, dtype=self.dtype).contiguous()
        if self.v_stored != e:               # zero columns where the stored heads have their extra columns
            wide = torch.zeros((W, H, self.v_stored), dtype=o.dtype, device=o.device)
            wide[:, :, :e] = o.view(W, H, e)
            o = wide.view(W, H * self.v_stored)
        self.o.load([o])
        if self.to_heads is not None:
            ks, vs = self.k_stored, self.v_stored
            keys = torch.zeros((H, ks, self.row), dtype=self.dtype, device=self.device)
            keys[:, :d, :n] = self.uk.view(H, d, n)
            keys[:, d:d + r, n:n + r] = torch.eye(r, dtype=self.dtype, device=self.device)
            values = torch.zeros((H, vs, self.row), dtype=self.dtype, device=self.device)
            values[:, :e, :n] = self.uv.view(H, e, n)
            self.to_heads.load([keys.view(H * ks, self.row), values.view(H * vs, self.row)])

    def _linear(self, writes_cache: bool) -> Linear:
        if writes_cache and not self.own_latent:
            raise ValueError("this latent attention layer has no latent of its own: it must read another place's cache")
        return self.proj if writes_cache else self.q_only

    def scratch_to_clear(self, ctx, tokens: int, writes_cache: bool = True) -> Optional[torch.Tensor]:
        """The projections' float32 buffer, if this step's product adds slices of K into it (decode-sized steps):
        the launch before this mixer clears it in passing."""
        lin = self._linear(writes_cache)
        if lin is None or not lin.meets_by_adds(tokens, torch.float32):
            return None
        buf = ctx.workspace.get("latent_proj", (tokens, lin.out_features), torch.float32)
        return buf if buf.numel() % 4 == 0 else None

    def _as_heads(self, ctx) -> bool:
        """Whether a prompt step makes keys and values per head instead of working in the latents' space."""
        if self.to_heads is None or ctx.is_decode or ctx.kv_total * self.heads_width * 2 > _HEADS_MAX_BYTES:
            return False
        if ctx.n_tokens * self.nh * self.row * 2 > _LATENT_MAX_BYTES:
            return True
        if self.prompt_way is not None:
            return self.prompt_way == "heads"
        seen = ctx.n_tokens * max(1.0, (ctx.kv_total - 0.5 * ctx.n_tokens) / ctx.n_seqs)     # (query, key) pairs, about
        heads = (_HEADS_FIXED_US + 2.0 * ctx.kv_total * self.heads_width * self.row / _PRODUCT_FLOPS_PER_US
                 + 2.0 * seen * self.heads_width / _HEADS_FLOPS_PER_US)
        latents = 2.0 * seen * self.nh * (self.row + self.rank) / _LATENT_FLOPS_PER_US
        return heads < latents

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx, cache_view, writes_cache: bool = True,
                scratch_cleared: bool = False) -> None:
        T = x.shape[0]
        ws = ctx.workspace
        group = cache_view.group
        lin = self._linear(writes_cache)
        proj = ws.get("latent_proj", (T, lin.out_features), torch.float32)
        lin.forward(x, proj, y_is_zero=scratch_cleared)
        table = self.position.fused_rotary_table() if self.position is not None else None
        gate = proj[:, self.gate_col:self.row_col] if self.gate else None
        row = (self.row_col, self.rank, self.row, self.norm_weight, self.eps, group.dest_rows, cache_view.k) \
            if writes_cache else None
        out = ws.get("latent_heads_out", (T, self.nh * self.v_stored), self.dtype)
        as_heads = self._as_heads(ctx)
        # sequences that begin with this step: their rows are the step's own, in the step's order
        rows = None
        if as_heads:
            rows = ws.get("latent_rows", (ctx.kv_total, self.row), self.dtype)
        fresh = as_heads and row is not None and ctx.kv_total == T
        if self.q_rank is not None:
            # the queries by way of their latent; the same launch finishes the token's row
            proj = self._queries_from_latent(proj, table, row, rows if fresh else None, ctx)
            row = None
        if as_heads:
            self._attend_as_heads(proj, table, row, rows, fresh, gate, out, ctx, cache_view)
        else:
            self._attend_latents(proj, table, row, gate, out, ctx, cache_view)
        self.o.forward_add(out, residual)

    def _queries_from_latent(self, proj, table, row, rows, ctx) -> torch.Tensor:
        T, ws = proj.shape[0], ctx.workspace
        q = ws.get("latent_q_proj", (T, self.q_width), torch.float32)
        clear = q if self.uq.meets_by_adds(T, torch.float32) and q.numel() % 4 == 0 else None
        a = ws.get("latent_q_down", (T, self.q_rank), self.dtype)
        ops.latent_down(proj, self.q_rank, self.q_norm_weight, self.eps, a, self.rot, table, ctx.positions, row, rows, clear)
        self.uq.forward(a, q, y_is_zero=clear is not None)
        return q

    def _attend_latents(self, proj, table, row, gate, out, ctx, cache_view) -> None:
        T, ws, group = proj.shape[0], ctx.workspace, cache_view.group
        H, n = self.nh, self.rank
        q = ws.get("latent_q", (T, H * self.row), self.dtype)
        ops.latent_queries(proj, 0, H, self.dim, self.rot, n, self.row, self.uk, table, ctx.positions, q, row)
        o = ws.get("latent_o", (T, H * n), self.dtype)
        partial = None
        if self.dtype == torch.float32:
            ops.attention_f32(q, cache_view.k, cache_view.k, o, group.block_table, ctx.token_seq, ctx.positions, H, 1,
                              self.row, group.page_size, 0, self.scale, vd=n)
        else:
            partial = ops.latent_attention(q, cache_view.k, o, group.block_table, ctx.q_start, ctx.kv_len, ctx.n_seqs,
                                           ctx.max_q_len, H, self.row, n, group.page_size, self.scale, ws,
                                           ctx.max_kv_len_bound)
        ops.latent_values(o, partial, self.uv, gate, out, H, n, self.vdim, self.v_stored)

    def _attend_as_heads(self, proj, table, row, rows, fresh, gate, out, ctx, cache_view) -> None:
        T, ws, group = proj.shape[0], ctx.workspace, cache_view.group
        H, ks, vs = self.nh, self.k_stored, self.v_stored
        q = ws.get("latent_q_heads", (T, H * ks), self.dtype)
        ops.latent_heads(proj, 0, H, self.dim, self.rot, ks, table, ctx.positions, q, row,
                         rows if fresh and row is not None else None)
        if not fresh:
            ops.gather_rows(cache_view.k, group.block_table, ctx.kv_len, ctx.kv_start, rows, group.page_size, ctx.n_seqs)
        kv = ws.get("latent_kv", (ctx.kv_total, self.heads_width), self.dtype)
        self.to_heads.forward(rows, kv)
        ops.attention_tc_matrix(q, kv, out, ctx.kv_start, ctx.q_start, ctx.kv_len, ctx.n_seqs, ctx.max_q_len, H, ks, vs,
                                ctx.max_kv_len_bound, self.scale, gate=gate if self.head_gate else None)
        if gate is not None and not self.head_gate:
            ops.sigmoid_gate(out, gate, H, self.vdim, vs)


register_part("mixer", "rotary_latent_attention", RotaryLatentAttention)

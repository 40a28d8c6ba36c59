"""Grouped-query softmax attention with capped scores, a chunked mask and an output gate, over the paged cache.

With h the mixer's input: q = Wq h (heads x dim), k = Wk h (kv_heads x dim), v = Wv h (kv_heads x vdim), no biases;
query head i uses key/value head floor(i / (heads / kv_heads)).  Every head of q and k is divided by its own root mean
square over dim (eps inside the root) and multiplied by a weight of size dim that the heads share; rotary positions
turn the first `rotary_dims` dimensions of every head of q and k (pairing i with i + rotary_dims / 2).  The score
(q . k) * scale becomes softcap * tanh(score / softcap) (softcap 0: as it is); position i sees j <= i with
floor(i / chunk) = floor(j / chunk), chunks counted from the sequence's first position (chunk 0: every j <= i);
ordinary softmax.  The concatenated heads are multiplied by sigmoid(Wg h) and projected by Wo.

Options that other designs use: `qk_norm` "unit" divides the heads of q and k by their root mean square without a
weight (after the rotation, which does not change a head's sum of squares, so the division is done on the way in);
`q_temp` (coef, every) multiplies the query at position p by 1 + coef ln(floor((p + 1) / every) + 1), a temperature
that grows with the sequence; `sink` adds one to the softmax's denominator, p_j = exp(s_j) / (1 + sum exp(s_j)): a key
of score 0 that has no value, so a query may attend to nothing; `sink` "learned" makes that score a number per head,
p_j = exp(s_j) / (exp(sink_h) + sum exp(s_j)); `slopes` (one per query head) takes slopes[h] (i - j) off the score of
position i with key j; `gate` "head": one number per head, sigmoid(Wg h)_h times the head's output; `value_mix`: in the
place named "first" the values are as projected and are left for later places of the step, in a place named "mix" the
values are (1 - vmix) v + vmix v_first with the first place's values of the same token, and that is what is cached.

q, k, v and the gate are one stacked product whose float32 accumulators one kernel turns into the queries and the
cache rows (`ops.head_norm_rope_cache`); the attention itself is the library's grouped-query attention (tcgen05 for
prompts, split keys for single tokens) with the cap, the chunk, the slopes, the sinks and a gate per head as arguments.
Single tokens of layers that neither norm nor turn their queries and keys skip that kernel: the attention kernel takes the
accumulators, mixes the values and appends the new key and value itself.  Keys are stored with a size of at least that of
the values (extra columns are zero: scores do not change), values with their own.  A chunk lets the cache give pages back.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch

from ..kernels import ops
from .attention import _FUSED_DECODE, _check_kernel_limits, stored_head_size
from .base import KVSpec, Mixer, PartSpec, register_part, shared_part
from .linear import Linear


FIRST_VALUES = "first_values"       # the step's shared tensor of a place with `value_mix` "first"


class CappedAttention(Mixer):
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float,
                 eps: float, softcap: float = 0.0, chunk: int = 0, qk_norm=True, gate=True,
                 position: Optional[PartSpec] = None, rotary_dims: int = 0, sink=False,
                 q_temp: Optional[tuple] = None, slopes: Optional[Sequence[float]] = None,
                 value_mix: Optional[str] = None,
                 dtype: torch.dtype = torch.bfloat16, device: torch.device = torch.device("cuda")):
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} heads are not a multiple of {num_kv_heads} key/value heads")
        if position is not None and (rotary_dims % 2 or not 0 < rotary_dims <= dim):
            raise ValueError(f"{rotary_dims} rotated dimensions do not fit vectors of size {dim}")
        if softcap < 0.0 or chunk < 0:
            raise ValueError(f"a cap ({softcap}) and a chunk ({chunk}) cannot be negative")
        self.hidden_size, self.nh, self.nkv = int(hidden_size), int(num_heads), int(num_kv_heads)
        self.dim, self.vdim = int(dim), int(vdim)
        self.scale, self.eps, self.softcap, self.chunk = float(scale), float(eps), float(softcap), int(chunk)
        if qk_norm not in (True, False, "unit"):
            raise ValueError(f"qk_norm is True (with weights), False or 'unit' (without), got {qk_norm!r}")
        self.unit_norm = qk_norm == "unit"
        if gate not in (True, False, "head") or sink not in (True, False, "learned"):
            raise ValueError(f"a gate is True, False or 'head', a sink True, False or 'learned', got {gate!r}, {sink!r}")
        if value_mix not in (None, "first", "mix"):
            raise ValueError(f"value_mix is None, 'first' or 'mix', got {value_mix!r}")
        if slopes is not None and softcap > 0.0:
            raise ValueError("scores are capped or take a distance bias, not both")
        if slopes is not None and len(slopes) != num_heads:
            raise ValueError(f"{len(slopes)} slopes do not fit {num_heads} heads")
        self.qk_norm, self.gate, self.head_gate = qk_norm is True, gate is not False, gate == "head"
        self.sink, self.learned_sink = sink is True, sink == "learned"
        self.value_mix, self.vmix = value_mix, 0.0
        self.slope_values, self.slopes, self.sinks = slopes, None, None
        self.temp_coef, self.temp_every = (0.0, 0) if q_temp is None else (float(q_temp[0]), int(q_temp[1]))
        if self.temp_every < 0:
            raise ValueError(f"a query temperature steps every {self.temp_every} positions")
        self.dtype, self.device = dtype, device
        self.v_stored = stored_head_size(self.vdim, dtype)
        self.k_stored = stored_head_size(self.dim, dtype)
        if dtype == torch.bfloat16:             # the tensor-core prompt kernel takes values up to the keys' size
            self.k_stored = max(self.k_stored, self.v_stored)
        _check_kernel_limits(self.nh, self.nkv, max(self.k_stored, self.v_stored), dtype)
        self.position = shared_part("position", position, dtype, device) if position is not None else None
        self.rotary_dims = int(rotary_dims) if position is not None else 0
        self.q_width, self.k_width, self.v_width = self.nh * self.dim, self.nkv * self.dim, self.nkv * self.vdim
        self.o_width = self.nh * self.vdim
        self.v_col = self.q_width + self.k_width
        self.gate_col = self.v_col + self.v_width
        self.gate_width = (self.nh if self.head_gate else self.o_width) if self.gate else 0
        self.proj = Linear(hidden_size, self.gate_col + self.gate_width, dtype, device, name="qkvg", pad_width=True)
        self.o = Linear(self.nh * self.v_stored, hidden_size, dtype, device, name="o", pad_width=True)
        self.wq = self.wk = None
        # single tokens: the attention kernel itself makes queries and cache rows from the accumulators
        self.fuses_decode = (dtype == torch.bfloat16 and _FUSED_DECODE and qk_norm is False and self.position is None
                             and self.temp_every == 0 and self.k_stored == self.dim and self.v_stored == self.vdim)

    def cache_spec(self) -> KVSpec:
        return KVSpec(self.nkv, self.k_stored, value_dim=0 if self.v_stored == self.k_stored else self.v_stored,
                      chunk=self.chunk)

    def limit_positions(self, n: int) -> None:
        limit = getattr(self.position, "limit_positions", None)
        if limit is not None:
            limit(n)

    def weight_shapes(self):
        shapes = {"q": ((self.q_width, self.hidden_size), "normal"), "k": ((self.k_width, self.hidden_size), "normal"),
                  "v": ((self.v_width, self.hidden_size), "normal"), "o": ((self.hidden_size, self.o_width), "normal")}
        if self.qk_norm:
            shapes.update(q_norm=((self.dim,), "ones"), k_norm=((self.dim,), "ones"))
        if self.gate:
            shapes["g"] = ((self.gate_width, self.hidden_size), "normal")
        if self.learned_sink:
            shapes["sink"] = ((self.nh,), "normal")
        if self.value_mix == "mix":
            shapes["vmix"] = ((), "normal")
        return shapes

    def load(self, q, k, v, o, q_norm=None, k_norm=None, g=None, sink=None, vmix=None) -> None:
        self.proj.load([q, k, v] + ([g] if self.gate else []))
        if tuple(o.shape) != (self.hidden_size, self.o_width):
            raise ValueError(f"weight 'o' of shape {tuple(o.shape)} does not fit ({self.hidden_size}, {self.o_width})")
        if self.v_stored != self.vdim:           # zero columns where the stored heads have their extra columns
            wide = torch.zeros((self.hidden_size, self.nh, self.v_stored), dtype=o.dtype, device=o.device)
            wide[:, :, : self.vdim] = o.view(self.hidden_size, self.nh, self.vdim)
            o = wide.view(self.hidden_size, self.nh * self.v_stored)
        self.o.load([o])
        if self.qk_norm:
            for t in (q_norm, k_norm):
                if tuple(t.shape) != (self.dim,):
                    raise ValueError(f"a head norm weight of shape {tuple(t.shape)} does not fit ({self.dim},)")
            self.wq = q_norm.to(device=self.device, dtype=torch.float32).contiguous()
            self.wk = k_norm.to(device=self.device, dtype=torch.float32).contiguous()
        if self.slope_values is not None:
            self.slopes = torch.tensor([float(s) for s in self.slope_values], dtype=torch.float32).to(self.device)
        if self.learned_sink:
            if tuple(sink.shape) != (self.nh,):
                raise ValueError(f"sinks of shape {tuple(sink.shape)} do not fit {self.nh} heads")
            self.sinks = sink.to(device=self.device, dtype=torch.float32).contiguous()
        if self.value_mix == "mix":
            if vmix.numel() != 1:
                raise ValueError(f"a share of the first values of shape {tuple(vmix.shape)} is not one number")
            self.vmix = float(vmix)

    def _projections(self, ctx, tokens: int) -> torch.Tensor:
        # the place whose values others mix in has a buffer of its own, which lasts as long as the step
        name = "capped_proj_first" if self.value_mix == "first" else "capped_proj"
        return ctx.workspace.get(name, (tokens, self.proj.out_features), torch.float32)

    def _first_values(self, ctx, tokens: int) -> Optional[torch.Tensor]:
        if self.value_mix != "mix":
            return None
        first = ctx.shared.get(FIRST_VALUES)
        if first is None or tuple(first.shape) != (tokens, self.v_width):
            raise ValueError("no earlier place of the step left values that this place can mix in")
        return first

    def scratch_to_clear(self, ctx, tokens: int, writes_cache: bool = True) -> Optional[torch.Tensor]:
        """The projections' float32 buffer, if this step's product adds slices of K into it (decode-sized steps):
        the launch before this mixer clears it in passing."""
        if not self.proj.meets_by_adds(tokens, torch.float32):
            return None
        buf = self._projections(ctx, tokens)
        return buf if buf.numel() % 4 == 0 else None

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx, cache_view, writes_cache: bool = True,
                scratch_cleared: bool = False) -> None:
        if not writes_cache:
            raise ValueError("this attention writes its own keys and values; it cannot read another place's")
        T = x.shape[0]
        ws = ctx.workspace
        group = cache_view.group
        proj = self._projections(ctx, T)
        self.proj.forward(x, proj, y_is_zero=scratch_cleared)
        if self.value_mix == "first":
            ctx.shared[FIRST_VALUES] = proj[:, self.v_col: self.gate_col]
        first = self._first_values(ctx, T)
        table = self.position.fused_rotary_table() if self.position is not None else None
        D, E = self.k_stored, self.v_stored
        gate = proj[:, self.gate_col:] if self.gate else None
        heads = dict(chunk=self.chunk, softcap=self.softcap, sink=self.sink, vd=E, slopes=self.slopes, sinks=self.sinks,
                     gate=gate if self.head_gate else None)
        attn = ws.get("capped_attn", (T, self.nh * E), self.dtype)
        bound = min(ctx.max_kv_len_bound, self.chunk) if self.chunk else ctx.max_kv_len_bound
        if ctx.is_decode and self.fuses_decode:
            ops.attention_bf16_decode(None, cache_view.k, cache_view.v, attn, group.block_table, ctx.kv_len, self.nh,
                                      self.nkv, D, group.page_size, 0, self.scale, ws, bound, qkv=proj,
                                      dest=group.dest_rows, first=first, mix=self.vmix, **heads)
        else:
            q = ws.get("capped_q", (T, self.nh * D), self.dtype)
            ops.head_norm_rope_cache(proj, self.wq, self.wk, self.eps, table, self.rotary_dims, ctx.positions, q,
                                     group.dest_rows, cache_view.k, cache_view.v, self.nh, self.nkv, self.dim, self.vdim, D,
                                     group.page_size, unit_norm=self.unit_norm, temp_coef=self.temp_coef,
                                     temp_every=self.temp_every, stored_vdim=E, first=first, mix=self.vmix)
            if self.dtype == torch.float32:
                ops.attention_f32(q, cache_view.k, cache_view.v, attn, group.block_table, ctx.token_seq, ctx.positions,
                                  self.nh, self.nkv, D, group.page_size, 0, self.scale, **heads)
            elif ctx.is_decode:
                ops.attention_bf16_decode(q, cache_view.k, cache_view.v, attn, group.block_table, ctx.kv_len, self.nh,
                                          self.nkv, D, group.page_size, 0, self.scale, ws, bound, **heads)
            else:
                attend = (ops.attention_tc_prefill if ops.attention_tc_supported(self.nh, self.nkv, D)
                          else ops.attention_bf16_prefill)
                attend(q, cache_view.k, cache_view.v, attn, group.block_table, ctx.q_start, ctx.kv_len, ctx.n_seqs,
                       ctx.max_q_len, self.nh, self.nkv, D, group.page_size, 0, self.scale, **heads)
        if self.gate and not self.head_gate:
            ops.sigmoid_gate(attn, gate, self.nh, self.vdim, E)
        self.o.forward_add(attn, residual)


register_part("mixer", "capped_attention", CappedAttention)

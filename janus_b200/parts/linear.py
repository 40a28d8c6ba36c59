"""Matrix products y = x W^T with W stored [out, in] (no bias anywhere in the
architecture: crates/janus-engine/src/model/block.rs:239-276 looks none up).

The engine dtype picks the kernel: float32 runs the CUDA-core product (true
32-bit), bfloat16 runs the tcgen05 tensor-core product with float32
accumulation.  Three epilogues: store, add into the float32 residual stream,
and SiLU-gate (for a stacked gate/up weight).
"""
from __future__ import annotations

from typing import Sequence

import torch

from ..kernels import ops


def _to_engine(w: torch.Tensor, dtype: torch.dtype, device: torch.device) -> torch.Tensor:
    return w.to(device=device, dtype=dtype).contiguous()


def _check_width(in_features: int, dtype: torch.dtype) -> None:
    """The tensor-core product reads its operands by TMA, whose rows must be multiples of 16 bytes: refuse
    other widths when the model is built, not at the first step."""
    if dtype == torch.bfloat16 and in_features % 8 != 0:
        raise ValueError(f"a bfloat16 product over {in_features} input features is not supported (the width "
                         f"must be a multiple of 8); such a model runs with dtype float32")


class _PaddedOperand:
    """For a `Linear(pad_width=True)` whose width is no multiple of 8: the weight gets zero columns up to the next
    multiple when it is loaded, and every call copies its rows into a buffer of that width with zeros behind them
    (one small launch).  Buffers only grow and outgrown ones are kept, since a captured decode step holds their
    address."""

    def __init__(self, in_features: int, device: torch.device):
        self.width = (in_features + 7) // 8 * 8
        self.device = device
        self._buffers = []

    def weight(self, w: torch.Tensor) -> torch.Tensor:
        pad = torch.zeros((w.shape[0], self.width - w.shape[1]), dtype=w.dtype, device=w.device)
        return torch.cat([w, pad], dim=1).contiguous()

    def rows(self, x: torch.Tensor) -> torch.Tensor:
        T = x.shape[0]
        if not self._buffers or self._buffers[-1].shape[0] < T:
            rows = 64
            while rows < T:
                rows *= 2
            self._buffers.append(torch.empty((rows, self.width), dtype=torch.bfloat16, device=self.device))
        out = self._buffers[-1][:T]
        ops.pad_rows_bf16(x, out)
        return out


class Linear:
    """One weight matrix, possibly the row-wise stack of several tensors of the
    checkpoint (q, k, v stacked so that one product serves all three)."""

    def __init__(self, in_features: int, out_features: int, dtype: torch.dtype, device: torch.device,
                 name: str = "", pad_width: bool = False):
        """`pad_width`: a bfloat16 product over a width that is no multiple of 8 runs on zero-padded copies of its
        operands instead of being refused."""
        self._padded = None
        if pad_width and dtype == torch.bfloat16 and in_features % 8 != 0:
            self._padded = _PaddedOperand(in_features, device)
        else:
            _check_width(in_features, dtype)
        self.in_features, self.out_features = in_features, out_features
        self.dtype, self.device = dtype, device
        self.name = name     # what a profile of a step calls this product
        self.weight = None   # float32: [out, in] row-major; bfloat16: ops.PackedWeight

    def load(self, tensors: Sequence[torch.Tensor]) -> None:
        parts = [_to_engine(t, self.dtype, self.device) for t in tensors]
        w = parts[0] if len(parts) == 1 else torch.cat(parts, dim=0)
        if tuple(w.shape) != (self.out_features, self.in_features):
            raise ValueError(f"weight of shape {tuple(w.shape)} does not fit "
                             f"({self.out_features}, {self.in_features})")
        if self._padded is not None:
            w = self._padded.weight(w)
        # bfloat16 products stream their weights as packed tiles (ops.PackedWeight); float32 stays row-major
        self.weight = ops.pack_weight(w) if self.dtype == torch.bfloat16 else w

    def load_row_major(self, w: torch.Tensor) -> None:
        """A matrix that is already on the device in the engine dtype (a head tied to the embedding: the
        float32 engine uses the embedding's storage as it is, the bfloat16 engine a packed copy)."""
        if tuple(w.shape) != (self.out_features, self.in_features):
            raise ValueError(f"weight of shape {tuple(w.shape)} does not fit ({self.out_features}, {self.in_features})")
        if self._padded is not None:
            w = self._padded.weight(w)
        self.weight = ops.pack_weight(w) if self.dtype == torch.bfloat16 else w

    def first_rows(self, rows: int) -> "Linear":
        """The product with the first `rows` output features only (shares storage)."""
        sub = Linear(self.in_features, rows, self.dtype, self.device, self.name, pad_width=self._padded is not None)
        sub._padded = self._padded          # the same padded copies of the rows serve both
        sub.weight = self.weight.first_rows(rows) if self.dtype == torch.bfloat16 else self.weight[:rows]
        return sub

    def meets_by_adds(self, tokens: int, y_dtype: torch.dtype) -> bool:
        """Whether `forward` into a float32 `y` for this many tokens cuts K into slices that
        meet in `y` by atomic adds, so that `y` has to be zero beforehand."""
        return (self.dtype != torch.float32 and y_dtype == torch.float32
                and ops.split_k_for(tokens, self.out_features, self._k()) > 1)

    def _k(self) -> int:
        return self.in_features if self._padded is None else self._padded.width

    # y = x W^T, stored in y's dtype (engine dtype, or float32 for logits)
    def forward(self, x: torch.Tensor, y: torch.Tensor, y_is_zero: bool = False) -> None:
        if self._padded is not None:
            x = self._padded.rows(x)
        if self.dtype == torch.float32:
            ops.gemm_f32(x, self.weight, y, accumulate=False, label=self.name)
        elif self.meets_by_adds(x.shape[0], y.dtype):
            # few tokens and few output tiles: slices of K run as CTAs of their own and meet in y
            if y_is_zero:
                pass
            elif y.numel() % 4 == 0 and y.data_ptr() % 16 == 0:
                ops.zero_f32(y)
            else:
                y.zero_()
            ops.gemm_bf16(x, self.weight, y, mode="add", label=self.name)
        else:
            ops.gemm_bf16(x, self.weight, y, mode="store", label=self.name)

    # residual += x W^T, the sum made in float32
    def forward_add(self, x: torch.Tensor, residual: torch.Tensor) -> None:
        if self._padded is not None:
            x = self._padded.rows(x)
        if self.dtype == torch.float32:
            ops.gemm_f32(x, self.weight, residual, accumulate=True, label=self.name)
        else:
            ops.gemm_bf16(x, self.weight, residual, mode="add", label=self.name)


class ActivatedLinear(Linear):
    """out = act(x W^T) in the engine dtype (`activation`: a name of `ops.ACTIVATIONS`, "gelu" or "relu2"): in the product's
    own epilogue, or, where a decode-sized step would leave SMs idle with K uncut (and in float32), behind a plain
    product."""

    def __init__(self, in_features: int, out_features: int, dtype: torch.dtype, device: torch.device, name: str = "",
                 pad_width: bool = False, activation: str = "gelu"):
        super().__init__(in_features, out_features, dtype, device, name, pad_width)
        if activation not in ops.ACTIVATIONS:
            raise ValueError(f"activation '{activation}' is not one of {sorted(ops.ACTIVATIONS)}")
        self.activation = activation

    def _behind(self, T: int) -> bool:
        return T <= 64 and self.meets_by_adds(T, torch.float32)

    def scratch_to_clear(self, ctx, tokens: int):
        """The plain product's float32 result, if slices of K are added into it: the launch before may clear it."""
        if not self._behind(tokens):
            return None
        z = ctx.workspace.get("activation_in", (tokens, self.out_features), torch.float32)
        return z if z.numel() % 4 == 0 else None

    def forward(self, x: torch.Tensor, out: torch.Tensor, ctx, scratch_cleared: bool = False) -> None:
        T = x.shape[0]
        if self.dtype == torch.float32 or self._behind(T):
            z = ctx.workspace.get("activation_in", (T, self.out_features), torch.float32)
            super().forward(x, z, y_is_zero=scratch_cleared)
            ops.activate(z, out, self.activation)
            return
        if self._padded is not None:
            x = self._padded.rows(x)
        ops.gemm_bf16(x, self.weight, out, mode=self.activation, label=self.name)


class GatedLinear:
    """out = silu(x Wg^T) * (x Wu^T) with Wg stacked over Wu
    (crates/janus-engine/src/model/block.rs:383-430).  With `limit` > 0 the activation is the clamped form
    g * sigmoid(alpha g) * (u + 1), g = min(x Wg^T, limit), u = clamp(x Wu^T, -limit, limit), in the same places:
    the product's own epilogue, or the activation kernel behind a plain product.  A negative `limit`
    (`ops.GELU_TANH_GATE`) makes the activation the tanh form of GELU on the gate: gelu_tanh(x Wg^T) * (x Wu^T)."""

    def __init__(self, in_features: int, out_features: int, dtype: torch.dtype, device: torch.device,
                 name: str = "gate_up", limit: float = 0.0, alpha: float = 1.0, pad_width: bool = False):
        self._padded = None
        if pad_width and dtype == torch.bfloat16 and in_features % 8 != 0:
            self._padded = _PaddedOperand(in_features, device)      # as `Linear(pad_width=True)`
        else:
            _check_width(in_features, dtype)
        self.limit, self.alpha = float(limit), float(alpha)
        self.in_features, self.out_features = in_features, out_features
        self.dtype, self.device = dtype, device
        self.name = name
        self.weight = None   # float32: [2 * out, in] row-major; bfloat16: a packed gated pair
        self._stacked = None  # bfloat16: the same tiles as one plain matrix (gate rows, then up rows)

    def load(self, gate: torch.Tensor, up: torch.Tensor) -> None:
        g, u = _to_engine(gate, self.dtype, self.device), _to_engine(up, self.dtype, self.device)
        for t in (g, u):
            if tuple(t.shape) != (self.out_features, self.in_features):
                raise ValueError(f"gate/up weight of shape {tuple(t.shape)} does not fit "
                                 f"({self.out_features}, {self.in_features})")
        if self._padded is not None:
            g, u = self._padded.weight(g), self._padded.weight(u)
        self.weight = ops.pack_gated(g, u) if self.dtype == torch.bfloat16 else torch.cat([g, u], dim=0)
        self._stacked = None

    def forward(self, x: torch.Tensor, out: torch.Tensor, ctx) -> None:
        if self._padded is not None:
            x = self._padded.rows(x)
        if self.dtype == torch.float32:
            gu = ctx.workspace.get("gate_up", (x.shape[0], 2 * self.out_features), torch.float32)
            ops.gemm_f32(x, self.weight, gu, accumulate=False, label=self.name)
            if self.limit != 0.0:
                ops.clamped_glu(gu, out, self.out_features, self.limit, self.alpha)
            else:
                ops.swiglu(gu, out)
        elif ops.gated_runs_unfused(x.shape[0], self.out_features):
            # few tokens, narrow layer: twice the tiles stream the weights as a plain product; the gate is applied after
            if self._stacked is None:
                self._stacked = self.weight.stacked()
            gu = ctx.workspace.get("gate_up", (x.shape[0], self._stacked.rows), torch.float32)
            ops.gemm_bf16(x, self._stacked, gu, mode="store", pair=False, label=self.name)
            if self.limit != 0.0:
                ops.clamped_glu(gu, out, 128 * self.weight.up_tile_offset, self.limit, self.alpha)
            else:
                ops.swiglu_f32_to_bf16(gu, out, 128 * self.weight.up_tile_offset)
        else:
            ops.gemm_bf16(x, self.weight, out, mode="swiglu", label=self.name, gate_limit=self.limit,
                          gate_alpha=self.alpha)

"""RMSNorm: y = x / sqrt(mean(x^2) + eps) * gamma, statistics in float32
(crates/janus-engine/src/compute/shaders/activations.wgsl:81-133).  The weight
keeps the dtype it was stored in (the reference keeps 1-D tensors in f32,
crates/janus-engine/src/compute/engine.rs:448-470), or is float32 when a constant is added to it (`weight_offset`: designs
that store a norm's weight around zero)."""
from __future__ import annotations

from typing import Optional

import torch

from ..kernels import ops
from .base import Norm, register_part


class RMSNorm(Norm):
    def __init__(self, width: int, eps: float, weight_offset: float = 0.0, dtype: torch.dtype = torch.bfloat16,
                 device: torch.device = torch.device("cuda")):
        self.width, self.eps, self.offset = int(width), float(eps), float(weight_offset)
        self.dtype, self.device = dtype, device
        self.gamma: Optional[torch.Tensor] = None

    def weight_shapes(self):
        return {"gamma": ((self.width,), "normal" if self.offset else "ones")}

    def load(self, gamma: torch.Tensor) -> None:
        if tuple(gamma.shape) != (self.width,):
            raise ValueError(f"norm weight of shape {tuple(gamma.shape)} does not fit ({self.width},)")
        if self.dtype == torch.float32 or self.offset:
            gamma = gamma.to(torch.float32)
        if self.offset:
            gamma = gamma + self.offset
        self.gamma = gamma.to(self.device).contiguous()

    def forward(self, x: torch.Tensor, out: torch.Tensor, row_index: Optional[torch.Tensor] = None,
                clear: Optional[torch.Tensor] = None) -> None:
        """`clear`: a float32 scratch tensor of the part that runs next, set to zero by the same launch."""
        ops.rmsnorm(x, self.gamma, self.eps, out, row_index, clear)

    def add_normed(self, y: Optional[torch.Tensor], residual: torch.Tensor, mult: float,
                   x_out: Optional[torch.Tensor] = None, clear: Optional[torch.Tensor] = None,
                   clear2: Optional[torch.Tensor] = None) -> None:
        """residual += mult * norm(y), y <- 0, x_out = residual in its dtype (y None: only that), one launch."""
        ops.sublayer_norm_add(y, self.gamma, self.eps, mult, residual, x_out, clear, clear2)

    def forward_streams(self, x: torch.Tensor, streams: int, weights: Optional[torch.Tensor], out: torch.Tensor,
                        row_index: Optional[torch.Tensor] = None, clear: Optional[torch.Tensor] = None,
                        clear2: Optional[torch.Tensor] = None) -> None:
        """The norm of the weighted sum of `streams` residual streams, summed and normed in one launch."""
        ops.streams_rmsnorm(x, streams, weights, self.gamma, self.eps, out, row_index, clear, clear2)


register_part("norm", "rms_norm", RMSNorm)


class LayerNorm(Norm):
    """y = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * gamma: a layer norm with a weight and no bias,
    statistics in float32 (the mean first, then the mean of the squared deviations)."""

    CENTER = True
    clears_two = True

    def __init__(self, width: int, eps: float, dtype: torch.dtype, device: torch.device):
        self.width, self.eps = int(width), float(eps)
        self.dtype, self.device = dtype, device
        self.gamma: Optional[torch.Tensor] = None

    def weight_shapes(self):
        return {"gamma": ((self.width,), "ones")}

    def load(self, gamma: torch.Tensor) -> None:
        if tuple(gamma.shape) != (self.width,):
            raise ValueError(f"norm weight of shape {tuple(gamma.shape)} does not fit ({self.width},)")
        self.gamma = gamma.to(device=self.device, dtype=torch.float32).contiguous()

    def forward(self, x: torch.Tensor, out: torch.Tensor, row_index: Optional[torch.Tensor] = None,
                clear: Optional[torch.Tensor] = None, clear2: Optional[torch.Tensor] = None) -> None:
        ops.join_norm(x, gamma=self.gamma, eps=self.eps, center=self.CENTER, x_out=out, row_index=row_index,
                      clear=clear, clear2=clear2)

    def join(self, residual: torch.Tensor, y: torch.Tensor, scale: Optional[torch.Tensor], out: torch.Tensor,
             clear2: Optional[torch.Tensor] = None) -> None:
        """residual += scale * y (per feature; None: y itself), y <- 0, out = norm(residual), in one launch."""
        ops.join_norm(residual, ya=y, scale=scale, gamma=self.gamma, eps=self.eps, center=self.CENTER, x_out=out,
                      clear2=clear2)


register_part("norm", "layer_norm", LayerNorm)


class DynamicTanh(Norm):
    """y = tanh(alpha * x) * gamma + beta feature by feature, alpha one number: an elementwise stand-in for a norm that
    needs no mean and no variance.  All in float32."""

    clears_two = True

    def __init__(self, width: int, dtype: torch.dtype, device: torch.device):
        self.width = int(width)
        self.dtype, self.device = dtype, device
        self.args: Optional[tuple] = None        # (gamma, beta, alpha) as the kernel takes them

    def weight_shapes(self):
        return {"gamma": ((self.width,), "ones"), "beta": ((self.width,), "normal"), "alpha": ((), "ones")}

    def load(self, gamma: torch.Tensor, beta: torch.Tensor, alpha: torch.Tensor) -> None:
        if tuple(gamma.shape) != (self.width,) or tuple(beta.shape) != (self.width,) or alpha.numel() != 1:
            raise ValueError(f"norm weights of shapes {tuple(gamma.shape)}, {tuple(beta.shape)}, {tuple(alpha.shape)} do "
                             f"not fit a width of {self.width}")
        f32 = lambda t: t.to(device=self.device, dtype=torch.float32).contiguous()     # noqa: E731
        self.args = (f32(gamma), f32(beta), float(alpha))

    def forward(self, x: torch.Tensor, out: torch.Tensor, row_index: Optional[torch.Tensor] = None,
                clear: Optional[torch.Tensor] = None, clear2: Optional[torch.Tensor] = None) -> None:
        ops.tanh_norm(x, norm_x=self.args, x_out=out, row_index=row_index, clear=clear, clear2=clear2)

    def add_normed(self, y: Optional[torch.Tensor], residual: torch.Tensor, mult: float,
                   x_out: Optional[torch.Tensor] = None, clear: Optional[torch.Tensor] = None,
                   clear2: Optional[torch.Tensor] = None) -> None:
        ops.tanh_norm(residual, y=y, norm_y=self.args, mult=mult, x_out=x_out, clear=clear, clear2=clear2)

    def add_normed_then(self, y: torch.Tensor, residual: torch.Tensor, mult: float, next_norm: Norm, x_out: torch.Tensor,
                        clear: Optional[torch.Tensor] = None) -> None:
        if not isinstance(next_norm, DynamicTanh):
            super().add_normed_then(y, residual, mult, next_norm, x_out, clear)
            return
        ops.tanh_norm(residual, y=y, norm_y=self.args, mult=mult, norm_x=next_norm.args, x_out=x_out, clear=clear)

    def replace(self, x: torch.Tensor) -> None:
        """x = norm(x) in place."""
        ops.tanh_norm(x, norm_y=self.args, replace=True)


register_part("norm", "dynamic_tanh", DynamicTanh)

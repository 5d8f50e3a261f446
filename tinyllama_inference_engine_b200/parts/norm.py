"""RMSNorm, with the residual add fused in front of it; the layer norm, with and without a bias; and the curve that may stand in a norm's place."""
from __future__ import annotations

import torch

from .. import ops
from .base import Norm, register_part
from .spec import PartSpec, TensorSpec


class RMSNorm(Norm):
    """y = x / sqrt(mean(x^2) + eps) * weight, eps inside the root (src/operators.cpp:22-45).

    params: ``size``, ``eps``, optional ``suffix`` (what follows the prefix in the tensor's name, ".weight" unless given), optional
    ``offset`` (the weight is stored minus this number: 1.0 for a weight stored around zero; added once, in 32-bit, at load time).
    tensors: ``<prefix><suffix> [size]``.
    The statistics, the scale and the residual sum are 32-bit in both precisions;
    the weight is held in 32-bit (exact for a bfloat16 checkpoint).
    """

    capturable = True
    supports_lazy = True

    @classmethod
    def tensor_specs(cls, spec: PartSpec, prefix: str) -> list[TensorSpec]:
        if float(spec.get("offset", 0.0) or 0.0) != 0.0:
            return [TensorSpec(f"{prefix}{spec.get('suffix', '.weight')}", (spec["size"],), init="matrix", std=0.1)]   # stored around zero
        return [TensorSpec(f"{prefix}{spec.get('suffix', '.weight')}", (spec["size"],), init="norm", std=0.1)]

    def __init__(self, spec, prefix, weights, runtime):
        super().__init__(spec, prefix, weights, runtime)
        self.size = int(spec["size"])
        self.eps = float(spec["eps"])
        self.weight = weights.get(f"{prefix}{spec.get('suffix', '.weight')}", torch.float32).contiguous()
        offset = float(spec.get("offset", 0.0) or 0.0)
        if offset != 0.0:
            self.weight = (self.weight + offset).contiguous()

    def forward(self, residual, delta=None, rows=None, lazy: bool = False):
        """``lazy`` (and nothing to add): hand the norm on to the product that consumes it (ops.LazyNorm)."""
        if lazy and delta is None:
            handle = ops.LazyNorm(residual, self.weight, self.eps, rows, lambda: self.forward(residual, None, rows))
            if rows is None and self.runtime.dtype == torch.bfloat16:
                # where a product that completes the residual may leave this norm's input (ops.linear_accumulate(..., prepare=handle))
                ws = self.runtime.workspace
                handle.buffers = (ws.get("prepared_norm", residual.shape[0], self.size, torch.bfloat16),
                                  ws.get("prepared_squares", residual.shape[0], -(-self.size // 16), torch.float32))
            return handle
        count = residual.shape[0] if rows is None else rows.shape[0]
        out = self.runtime.workspace.get("normed" if rows is None else "normed_rows", count, self.size, self.runtime.dtype)
        ops.add_rmsnorm(residual, delta, self.weight, self.eps, out, rows)
        return out


class LayerNorm(Norm):
    """y = (x - mean) / sqrt(mean((x - mean)^2) + eps) * weight (+ bias): a layer norm.

    params: ``size``, ``eps``, optional ``suffix`` (what follows the prefix in the tensor's name, ".weight" unless given), optional ``bias`` (whether there
    is a tensor of the same name with ".b" added).
    tensors: ``<prefix><suffix> [size]``, ``<prefix><suffix>.b [size]``.  Mean, variance, scale and the residual sum are 32-bit in both precisions; weight and
    bias are held in 32-bit.  ``forward`` adds ``delta`` into the stream first, as the RMS norm does; ``join`` is what a block calls that normalises a
    branch before it joins the stream: ``residual += self(y)``, and in the same kernel the next norm of the stream if one is named.
    ``join_stream`` is the same for a block whose next sublayer reads the stream itself.
    """

    capturable = True
    supports_lazy = False
    centred = True
    groups = 1

    @classmethod
    def tensor_specs(cls, spec: PartSpec, prefix: str) -> list[TensorSpec]:
        name = f"{prefix}{spec.get('suffix', '.weight')}"
        return [TensorSpec(name, (spec["size"],), init="norm", std=0.1)] + ([TensorSpec(f"{name}.b", (spec["size"],), std=0.2)] if spec.get("bias") else [])

    def __init__(self, spec, prefix, weights, runtime):
        super().__init__(spec, prefix, weights, runtime)
        self.size = int(spec["size"])
        self.eps = float(spec["eps"])
        name = f"{prefix}{spec.get('suffix', '.weight')}"
        self.weight = weights.get(name, torch.float32).contiguous()
        self.bias = weights.get(f"{name}.b", torch.float32).contiguous() if spec.get("bias") else None

    def forward(self, residual, delta=None, rows=None, lazy: bool = False):
        if delta is not None:
            ops.add_(residual, delta)
        count = residual.shape[0] if rows is None else rows.shape[0]
        out = self.runtime.workspace.get("normed" if rows is None else "normed_rows", count, self.size, self.runtime.dtype)
        ops.branch_norm(residual, None, None, self.weight, out, self.eps, self.centred, rows, groups=self.groups, next_bias=self.bias)
        return out

    def join(self, residual, branch, following: "LayerNorm | None" = None):
        """``residual += self(branch)``; with ``following`` (a norm of this kind and eps) also returns ``following(residual)``, one kernel."""
        if following is None:
            ops.branch_norm(residual, branch, self.weight, None, None, self.eps, self.centred, groups=self.groups, post_bias=self.bias)
            return None
        out = self.runtime.workspace.get("normed", residual.shape[0], self.size, self.runtime.dtype)
        ops.branch_norm(residual, branch, self.weight, following.weight, out, self.eps, self.centred, groups=self.groups, post_bias=self.bias, next_bias=following.bias)
        return out

    def join_stream(self, residual, branch):
        """``residual += self(branch)``; returns the finished stream as the next product's operand: rounded by the same kernel, or in the 32-bit
        path the stream itself."""
        if self.runtime.dtype == torch.float32:
            self.join(residual, branch)
            return residual
        out = self.runtime.workspace.get("stream_rounded", residual.shape[0], self.size, self.runtime.dtype)
        ops.branch_norm(residual, branch, self.weight, None, out, self.eps, self.centred, groups=self.groups, post_bias=self.bias)
        return out


class GroupedRMSNorm(LayerNorm):
    """y = x / sqrt(mean(x^2) + eps) * weight over each of ``groups`` equal consecutive parts of a row, every part with a root mean
    square of its own (one group: the plain RMS norm).

    params: ``size``, ``eps``, ``groups``, optional ``suffix`` and ``scale`` (the weight is multiplied by it once, in 32-bit, at load time:
    a branch that joins the stream times a constant).  ``forward`` and ``join`` are the layer norm's: the norm of a branch, its sum
    into the 32-bit stream and the stream's next norm are one kernel."""

    centred = False

    def __init__(self, spec, prefix, weights, runtime):
        super().__init__(spec, prefix, weights, runtime)
        self.groups = int(spec.get("groups", 1) or 1)
        if self.size % self.groups:
            from ..errors import ConfigError

            raise ConfigError(f"{prefix}: a norm over {self.size} columns cannot have {self.groups} equal groups")
        scale = float(spec.get("scale", 1.0))
        if scale != 1.0:
            self.weight = (self.weight * scale).contiguous()


class DynamicTanh(Norm):
    """y = tanh(alpha x) * weight + bias element by element: what stands in the place of a norm where no statistics are taken.

    params: ``size``, optional ``suffix`` (what follows the prefix in the tensor's name, ".weight" unless given).
    tensors: ``<prefix><suffix>`` [size], ``<prefix><suffix>.b`` [size], ``<prefix><suffix>.alpha`` [].  The residual sum, the curve, weight and bias are 32-bit.
    ``forward`` takes one output that is still to join the stream, as the other norms do; ``join`` takes up to two and hands the result over as an
    ``ops.FinishedNorm``.  Since an element's value needs nothing of its row, a product that completes the stream can leave this norm's output
    beside it (``pending``, ``ops.linear_accumulate``)."""

    capturable = True
    supports_lazy = False

    @classmethod
    def tensor_specs(cls, spec: PartSpec, prefix: str) -> list[TensorSpec]:
        name = f"{prefix}{spec.get('suffix', '.weight')}"
        return [TensorSpec(name, (spec["size"],), init="norm", std=0.1), TensorSpec(f"{name}.b", (spec["size"],), std=0.2), TensorSpec(f"{name}.alpha", (), init="uniform", std=1.0)]

    def __init__(self, spec, prefix, weights, runtime):
        super().__init__(spec, prefix, weights, runtime)
        self.size = int(spec["size"])
        name = f"{prefix}{spec.get('suffix', '.weight')}"
        self.weight = weights.get(name, torch.float32).contiguous()
        self.bias = weights.get(f"{name}.b", torch.float32).contiguous()
        self.alpha = float(weights.get(f"{name}.alpha", torch.float32))

    def _out(self, rows: int, name: str = "normed"):
        return self.runtime.workspace.get(name, rows, self.size, self.runtime.dtype)

    def forward(self, residual, delta=None, rows=None, lazy: bool = False):
        out = self._out(residual.shape[0]) if rows is None else self._out(rows.shape[0], "normed_rows")
        if rows is not None and delta is not None:
            ops.add_(residual, delta)
            delta = None
        ops.dynamic_tanh(residual, delta, None, rows, self.weight, self.bias, self.alpha, out)
        return out

    def pending(self, residual) -> "ops.FinishedNorm":
        """This norm of ``residual`` as it will be: for the product that completes it to finish."""
        buffer = self._out(residual.shape[0]) if self.runtime.dtype == torch.bfloat16 else None
        return ops.FinishedNorm(self, residual, (self.alpha, self.weight, self.bias), buffer)

    def join(self, residual, first, second=None) -> "ops.FinishedNorm":
        """``residual += first + second`` (either may be None) and this norm of the result, one kernel."""
        handle = ops.FinishedNorm(self, residual, (self.alpha, self.weight, self.bias), None)
        handle.finished = self._out(residual.shape[0])
        ops.dynamic_tanh(residual, first, second, None, self.weight, self.bias, self.alpha, handle.finished)
        return handle


register_part("norm", "dynamic_tanh", DynamicTanh)
register_part("norm", "grouped_rmsnorm", GroupedRMSNorm)
register_part("norm", "rmsnorm", RMSNorm)
register_part("norm", "layernorm", LayerNorm)

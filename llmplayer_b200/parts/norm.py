"""Norms of the residual stream, in float32: RMS norm, out = x / sqrt(mean(x^2) + eps) * gain, over whole rows or over
equal parts of a row (each with its own root mean square), and layer norm with a gain and no bias.

Reference: inference/RMSNorm.java:17-35, tensor/ScalarOps.java:26-35,
src/main/resources/kernels/cuda/rmsnorm.cu:6-46. The gain is used as stored.
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..errors import ConfigError
from ..kernels import ops
from .base import NORMS, Part, Runtime
from .specs import GAIN, NormSpec, TensorSpec


class RMSNorm(Part):
    capture_safe = True

    def __init__(self, spec: NormSpec):
        if spec.groups <= 0 or spec.size % spec.groups:
            raise ConfigError(f"a row of {spec.size} values cannot be normed in {spec.groups} equal parts")
        self.spec = spec
        self.rms_parts = spec.groups            # a kernel that norms the stream in so many equal parts may write this norm
        # a product that adds into the residual stream, or reads it, may apply this norm on the way (one factor per row)
        self.fusable_rms = spec.groups == 1
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {self.spec.weight: TensorSpec((self.spec.size,), GAIN)}

    def load(self, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().load(tensors, runtime)
        self.weight = runtime.gain(tensors[self.spec.weight])

    def apply(self, x: torch.Tensor, out: torch.Tensor, rows: Optional[torch.Tensor] = None,
              add: Optional[torch.Tensor] = None, clear: Optional[torch.Tensor] = None) -> torch.Tensor:
        """``out[r] = norm(x[rows[r]])``; ``add`` is summed into ``x`` first (in place);
        ``clear`` is a float32 buffer zeroed on the side."""
        return ops.rmsnorm(x, self.weight, self.spec.eps, out, rows=rows, add=add, clear=clear, parts=self.rms_parts)


class LayerNorm(Part):
    """out = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * gain, in float32; no bias."""
    capture_safe = True

    def __init__(self, spec: NormSpec):
        self.spec = spec
        self.weight: Optional[torch.Tensor] = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {self.spec.weight: TensorSpec((self.spec.size,), GAIN)}

    def load(self, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> None:
        super().load(tensors, runtime)
        self.weight = runtime.gain(tensors[self.spec.weight])

    def apply(self, x: torch.Tensor, out: torch.Tensor, rows: Optional[torch.Tensor] = None,
              add: Optional[torch.Tensor] = None, clear: Optional[torch.Tensor] = None) -> torch.Tensor:
        if add is not None:
            raise ConfigError("the layer norm kernel does not add a residual on the way")
        return ops.layernorm(x, self.weight, self.spec.eps, out, rows=rows, clear=clear)


NORMS.register("rmsnorm", RMSNorm)
NORMS.register("layernorm", LayerNorm)

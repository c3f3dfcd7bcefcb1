"""Normalisation parts."""

from __future__ import annotations

from .base import Norm, NormedInput, NormedUpdate
from .registry import NORMS
from .spec import TensorSpec


@NORMS.register("rmsnorm")
class RMSNorm(Norm):
    """v * rsqrt(mean(v^2) + eps) * weight over the last axis, computed in 32-bit, fused
    with the residual add that precedes it. Parameters: ``size``, ``eps``, ``offset`` (0; a
    weight stored around zero has offset 1 and the norm multiplies by offset + weight).
    Reference: nn.RMSNorm at src/mlx_one/models/language/lfm2/reference_math.py:156-157."""

    supports_lazy = True

    @classmethod
    def tensors(cls, spec):
        return {"weight": TensorSpec((spec["size"],), "norm0" if spec.get("offset") else "norm")}

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.weight = self.vector(tensors["weight"])
        if spec.get("offset"):
            self.weight = (self.weight + float(spec["offset"])).contiguous()
        self.eps = float(spec["eps"])

    def forward(self, residual, delta, lazy=False, delta_scale=1.0):
        can_fuse = getattr(self.ops, "can_fuse_norm", None)
        if lazy and delta is None and can_fuse is not None and can_fuse(residual, self.runtime.dtype):
            return NormedInput(residual, self.weight, self.eps, self.runtime.dtype, self.ops)
        if delta is None or delta_scale == 1.0:
            return self.ops.add_rmsnorm(residual, delta, self.weight, self.eps, self.runtime.dtype)
        return self.ops.add_rmsnorm(residual, delta, self.weight, self.eps, self.runtime.dtype,
                                    delta_scale=delta_scale)

    def read_streams(self, streams, update, read):
        """From parallel streams [tokens, n, hidden]: applies the pending ``update`` (a
        StreamUpdate or None) and norms u = sum_s read[s] X_s. Returns (the streams after the
        update, the normed u in the compute dtype)."""
        return self.ops.read_streams(streams, update, read, self.weight, self.eps,
                                     self.runtime.dtype)

    def add_normed(self, residual, x):
        """In place: residual += x * rsqrt(mean(x^2) + eps) * weight, the norm taken over a part's
        output ``x`` (compute dtype) and everything in 32-bit."""
        self.ops.normed_mean_add(residual, [x], [self.weight], self.eps)


@NORMS.register("layernorm")
class LayerNorm(Norm):
    """(v - mean) * rsqrt(variance + eps) * weight + bias over the last axis, the variance being the
    mean of the squared deviations; 32-bit, fused with what is added to the stream before it: a
    plain output, or one that is normed itself (``NormedUpdate``). Parameters: ``size``, ``eps``."""

    @classmethod
    def tensors(cls, spec):
        return {"weight": TensorSpec((spec["size"],), "norm"), "bias": TensorSpec((spec["size"],), "bias")}

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.weight, self.bias = self.vector(tensors["weight"]), self.vector(tensors["bias"])
        self.eps = float(spec["eps"])

    def forward(self, residual, delta, lazy=False, delta_scale=1.0):
        return self.ops.add_norm(residual, delta, self.weight, self.bias, self.eps,
                                 self.runtime.dtype, delta_scale=delta_scale)

    def update(self, output):
        """residual + norm(output), still to be added."""
        return NormedUpdate(output, self.weight, self.bias, self.eps)

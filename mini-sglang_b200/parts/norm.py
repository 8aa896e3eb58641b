from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..weights.loader import TensorDecl
from .base import NORMS, Norm, build_part, register_norm


@register_norm("rmsnorm")
class RMSNorm(Norm):
    """y = v * rsqrt(mean(v^2) + eps) * weight (+ bias) with v = residual + x, in float32; plain weight.
    Formula of mini_sglang/layers/layernorm.py:39-50.  params: size, eps, optional name
    (full tensor name; default "<prefix>.weight"), bias (False; the tensor is "<name>.b")."""

    center = False        # whether the row's mean is taken off first

    def __init__(self, spec, prefix, env):
        super().__init__(spec, prefix, env)
        self.size, self.eps = int(spec["size"]), float(spec["eps"])
        self.tensor_name = spec.get("name") or self.name("weight")
        self.has_bias = bool(spec.get("bias", False))
        self.weight = self.bias = None

    def tensors(self) -> Dict[str, TensorDecl]:
        t = {self.tensor_name: TensorDecl((self.size,), kind="vector", init="norm")}
        if self.has_bias:
            t[self.tensor_name + ".b"] = TensorDecl((self.size,), kind="vector", std=0.1)
        return t

    def load(self, src) -> None:
        self.weight = src.fetch(self.tensor_name).contiguous()
        if self.has_bias:
            self.bias = src.fetch(self.tensor_name + ".b").float().contiguous()

    def forward(self, x=None, residual=None, residual_out=None, rows=None):
        return ops.rmsnorm(self.weight, self.eps, x=x, residual=residual, residual_out=residual_out, rows=rows,
                           out_dtype=self.env.dtype, center=self.center, bias=self.bias)

    def fused_decode_fields(self):
        if self.center or self.has_bias:
            return None
        return {"kind": "rmsnorm", "weight": self.weight, "eps": self.eps, "size": self.size}


@register_norm("layernorm")
class LayerNorm(RMSNorm):
    """y = (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps) * weight (+ bias) with v = residual + x, in float32.
    params as `rmsnorm`."""

    center = True


@register_norm("dynamic_tanh")
class DynamicTanh(Norm):
    """y = tanh(alpha * v) * weight + bias with v = residual + x in float32, element by element: a norm that takes no mean
    and no variance of the row.  Tensors: the weight under `name` (default "<prefix>.weight"), the bias under "<name>.b" and
    the scalar alpha under "<name>.alpha".  params: size, optional name."""

    def __init__(self, spec, prefix, env):
        super().__init__(spec, prefix, env)
        self.size = int(spec["size"])
        self.tensor_name = spec.get("name") or self.name("weight")
        self.weight = self.bias = None
        self.alpha = 1.0

    def tensors(self) -> Dict[str, TensorDecl]:
        return {self.tensor_name: TensorDecl((self.size,), kind="vector", init="norm"),
                self.tensor_name + ".b": TensorDecl((self.size,), kind="vector"),
                self.tensor_name + ".alpha": TensorDecl((), kind="vector", init="norm")}

    def load(self, src) -> None:
        self.weight = src.fetch(self.tensor_name).float().contiguous()
        self.bias = src.fetch(self.tensor_name + ".b").float().contiguous()
        self.alpha = float(src.fetch(self.tensor_name + ".alpha").float().item())

    def forward(self, x=None, residual=None, residual_out=None, rows=None):
        return ops.dyntanh(self.weight, self.bias, self.alpha, x=x, residual=residual, residual_out=residual_out, rows=rows,
                           out_dtype=self.env.dtype)


@register_norm("stream_sum")
class StreamSumNorm(Norm):
    """The end of a model that keeps several copies of the residual stream: the copies as the last sublayer leaves them are
    added up and normed.  `residual` [T, S, H] holds the copies before that sublayer's update, `x` its pending update (a
    `parts.streams.StreamUpdate`); update, sum and norm are one kernel that touches the wanted rows only.
    params: norm (the PartSpec of an `rmsnorm` or `layernorm`), streams."""

    def __init__(self, spec, prefix, env):
        super().__init__(spec, prefix, env)
        self.norm = build_part(NORMS, "norm", spec["norm"], prefix, env)
        if not hasattr(self.norm, "center"):
            raise ValueError("the copies of the stream are summed into an RMS norm or a layer norm; another kind is not taken here")
        self.streams = int(spec["streams"])

    def tensors(self) -> Dict[str, TensorDecl]:
        return self.norm.tensors()

    def load(self, src) -> None:
        self.norm.load(src)
        self.weight = self.norm.weight.float().contiguous()

    def forward(self, x=None, residual=None, residual_out=None, rows=None):
        assert residual_out is None
        u = x
        return ops.stream_mix_norm(residual, streams=self.streams, weight=self.weight, bias=self.norm.bias, eps=self.norm.eps,
                                   center=self.norm.center, w_in=None, y=u.y if u is not None else None,
                                   mix=u.mix if u is not None else None, w_out=u.w_out if u is not None else None, rows=rows,
                                   out_dtype=self.env.dtype)

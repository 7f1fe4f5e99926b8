"""RMSNorm: y = x * (1 / sqrt(mean(x^2) + eps)) * w, statistics in 32-bit.

eps sits inside the square root and the weight multiplies last, with no bias and no "+1"
(src/model.rs:919-928, src/cuda.rs:505-515).

"dynamic_tanh": y = tanh(alpha x) * w + b, element by element, without mean or variance; alpha is one learned number.

"layernorm": y = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * w, with a weight and no bias, also 32-bit.

`forward(x, rows=None, out_dtype=None)`: `out_dtype` None is the step's activation type; a model that norms its
embeddings asks for float32, the stream's own type.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernels import ops
from .base import Norm, RowRead, StreamRead, WeightSpec
from .registry import register


@register("norm", "rmsnorm")
class RmsNorm(Norm):
    settles_pending = True      # its kernel adds partial sums a deferred product left for the rows it reads

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.size = int(params["size"])
        self.eps = float(params["eps"])

    def weights(self) -> List[WeightSpec]:
        return [WeightSpec(self.tensor_name("weight", "weight"), (self.size,), "ones")]

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        self.weight = rt.place(tensors[self.tensor_name("weight", "weight")])
        self._weight32 = None

    @property
    def weight32(self) -> torch.Tensor:
        """The weight as 32-bit values (what joins the residual sum is 32-bit), made when first asked for."""
        if self._weight32 is None:
            self._weight32 = self.weight.to(torch.float32).contiguous()
        return self._weight32

    def row_read(self, step):
        return RowRead(self.weight, self.eps, self.rt.dtype)

    def forward(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
        if rows is None:
            h = ops.take_handed(x, self)
            if h is not None and h.dtype == (out_dtype or self.rt.dtype):
                return h
        with ops.bucket("norm"):
            return ops.rmsnorm(x, self.weight, self.eps, out_dtype or self.rt.dtype, rows=rows)


    def add_normed(self, x: torch.Tensor, y: torch.Tensor, scale: Optional[torch.Tensor] = None,
                   cast_out: Optional[torch.Tensor] = None, zero_y: bool = False) -> None:
        """x += y / sqrt(mean(y^2) + eps) * w [* scale]: the norm on a sublayer's output, joined to the stream in one pass;
        the same pass can leave the new stream in the activation type in `cast_out` and y zeroed, for the next sublayer."""
        with ops.bucket("norm"):
            ops.postnorm_add(x, y, self.weight32, self.eps, scale, cast_out=cast_out, zero_y=zero_y)


@register("norm", "channel_scale")
class ChannelScale(Norm):
    """A learned number per channel that multiplies a sublayer's normed output (kept 32-bit: it joins the residual sum)."""

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.size = int(params["size"])

    def weights(self) -> List[WeightSpec]:
        return [WeightSpec(self.tensor_name("weight", "weight"), (self.size,), "ones")]

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        self.weight = tensors[self.tensor_name("weight", "weight")].to(device=rt.device, dtype=torch.float32).contiguous()

    def forward(self, x, rows=None, out_dtype=None):
        raise NotImplementedError("a channel scale is applied by the block that holds it")


@register("norm", "layernorm")
class LayerNorm(Norm):
    settles_pending = True      # its kernel adds partial sums a deferred product left for the rows it reads

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.size = int(params["size"])
        self.eps = float(params["eps"])

    def weights(self) -> List[WeightSpec]:
        return [WeightSpec(self.tensor_name("weight", "weight"), (self.size,), "ones")]

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        self.weight = rt.place(tensors[self.tensor_name("weight", "weight")])

    def forward(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
        with ops.bucket("norm"):
            return ops.layernorm(x, self.weight, self.eps, out_dtype or self.rt.dtype, rows=rows)


@register("norm", "dynamic_tanh")
class DynamicTanh(Norm):
    """y = tanh(alpha * x) * w + b (32-bit).  Tensors: the prefix + "weight", "b", "alpha" unless `params["tensor_names"]` gives
    others for the keys "weight", "bias", "alpha".  Nothing about it spans a row, so it rides in the pass that writes the stream:
    `join` adds a normed sublayer output to the stream and does the next reader's operation on the way."""
    settles_pending = True

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.size = int(params["size"])
        self.names = {k: self.tensor_name(k, v) for k, v in {"weight": "weight", "bias": "b", "alpha": "alpha"}.items()}

    def weights(self) -> List[WeightSpec]:
        n = self.names
        return [WeightSpec(n["weight"], (self.size,), "ones"), WeightSpec(n["bias"], (self.size,)), WeightSpec(n["alpha"], (), "ones")]

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        n = self.names
        # weights as 32-bit values: what they multiply joins 32-bit sums, and every norm of a pass then has the same type
        f32 = lambda name: tensors[name].to(device=rt.device, dtype=torch.float32).contiguous()
        self.weight, self.b = f32(n["weight"]), f32(n["bias"])
        self.alpha = float(tensors[n["alpha"]].to(torch.float32).reshape(-1)[0])
        self.numbers = (self.alpha, self.weight, self.b)

    def stream_read(self, step):
        return StreamRead(self.numbers, self.rt.dtype)

    def forward(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
        want = out_dtype or self.rt.dtype
        if rows is None:
            h = ops.take_handed(x, self)
            if h is not None and h.dtype == want:
                return h
        with ops.bucket("norm"):
            # sums pending for the stream stay in it, unless only chosen rows are read (whoever does that is its last reader)
            keep = x if rows is None and ops.has_pending(x) else None
            return ops.tanh_rows(x, None, None, self.numbers, want, rows=rows, x_out=keep, quick=self.rt.dtype != torch.float32)

    def start_stream(self, e: torch.Tensor, step) -> torch.Tensor:
        x = ops.as_carrier(e)
        self.join(None, x, step.next_reader, step, x_out=x)
        return x

    def join(self, x: Optional[torch.Tensor], y: torch.Tensor, reader, step, zero_y: bool = False, x_out: Optional[torch.Tensor] = None) -> None:
        """x += norm(y) (no x: the rows themselves, into `x_out`); y is zeroed if asked; and if `reader` (who reads the stream
        next, or None) can say what it does first, that is done in the same pass and left with the stream."""
        out = x if x is not None else x_out
        read = reader.stream_read(step) if reader is not None else None
        with ops.bucket("norm"):
            h = ops.tanh_rows(x, y, self.numbers, read.norm if read is not None else None, read.dtype if read is not None else None,
                              x_out=out, base=read.base if read is not None else None, zero_y=zero_y, quick=self.rt.dtype != torch.float32)
        if h is not None:
            ops.hand_on(out, reader, h)

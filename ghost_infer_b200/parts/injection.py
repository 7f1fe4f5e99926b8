"""What the stream passes through before every pass over a model's looped layers: x <- W [x; x0], x0 being the stream as the
embedding left it.

W is stored [width, 2 width] with the columns that read x first.  Its two halves are kept apart: W_0 x0 is the same for every
pass of a step, so it is formed once and each pass adds W_x x to it (in 32 bits).  Where the first pass comes right after the
embedding, x is x0 and one product over both halves stacked gives both sums.

Tensor name: the prefix itself unless `params["tensor_names"]` gives another for the key "weight".
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernels import ops
from .base import Injection, StreamRead, WeightSpec
from .linear import linear
from .registry import register


@register("injection", "input_injection")
class InputInjection(Injection):
    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.width = int(params["hidden_size"])
        self.name = self.tensor_name("weight", "")

    def weights(self) -> List[WeightSpec]:
        return [WeightSpec(self.name, (self.width, 2 * self.width))]

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        w, d = rt.place(tensors[self.name]), self.width
        self.w_both = torch.cat([w[:, :d], w[:, d:]], dim=0).contiguous()       # [W_x; W_0]
        self.w_x, self.w_0 = self.w_both[:d], self.w_both[d:]

    def _carried(self, step) -> Optional[torch.Tensor]:
        return step.shared.get((id(self), "carried"))

    def begin(self, x0, step, starts: bool) -> None:
        """W_0 x0 for the step; with `starts` also W_x x0, which the first `forward` then finds ready."""
        h = ops.take_handed(x0, self) if starts else None       # else what was left with the stream is for another reader
        if h is None:
            h = ops.cast_rows(x0, self.rt.dtype)
        with ops.bucket("out matmul"):
            if starts:
                both = linear(h, self.w_both, out_dtype=torch.float32)
                step.shared[(id(self), "first")] = both[:, :self.width]
                step.shared[(id(self), "carried")] = both[:, self.width:]
            else:
                step.shared[(id(self), "carried")] = linear(h, self.w_0, out_dtype=torch.float32)

    def stream_read(self, step):
        # before `begin` the embedding output itself has to stay in the stream; later passes start from W_0 x0
        return StreamRead(None, self.rt.dtype, self._carried(step))

    def forward(self, x, step) -> None:
        base, first = self._carried(step), step.shared.pop((id(self), "first"), None)
        if first is not None:                        # x <- W_x x0 + W_0 x0, and the next reader's norm on the way
            reader = step.next_reader
            read = reader.stream_read(step) if reader is not None else None
            with ops.bucket("norm"):
                h = ops.tanh_rows(first, base, None, read.norm if read else None, read.dtype if read else None, x_out=x,
                                  quick=self.rt.dtype != torch.float32)
            if h is not None:
                ops.hand_on(x, reader, h)
            return
        h = ops.take_handed(x, self)
        if h is None:                                # nobody did it on the way: the stream as the product reads it, then its new start
            with ops.bucket("norm"):
                h = ops.tanh_rows(x, None, None, None, self.rt.dtype, x_out=x, base=base)
        with ops.bucket("out matmul"), ops.defer_into(x):
            linear(h, self.w_x, out=x, accumulate=True)

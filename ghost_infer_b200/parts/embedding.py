"""Token embedding and output head.

x[t] = E[token_t] (src/model.rs:987-990), times `scale` where a model names one; logits = W normed with no bias and no cap (times
`scale` where a model names one; capped by c tanh(. / c) where it names a `softcap` c), where W is the embedding table when the model ties them (src/model.rs:637-638, :1183-1186).
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..kernels import ops
from ..cache.sequence_cache import StateRequest
from .base import Embedding, Part, WeightSpec
from .linear import linear
from .registry import register


@register("embedding", "token_embedding")
class TokenEmbedding(Embedding):
    def __init__(self, params, prefix="model.embed_tokens."):
        super().__init__(params, prefix)
        self.vocab = int(params["vocab_size"])
        self.hidden = int(params["hidden_size"])
        self.scale = float(params.get("scale", 1.0))

    def weights(self) -> List[WeightSpec]:
        return [WeightSpec(self.tensor_name("weight", "weight"), (self.vocab, self.hidden))]

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        self.weight = rt.place(tensors[self.tensor_name("weight", "weight")])

    def forward(self, tokens: torch.Tensor) -> torch.Tensor:
        with ops.bucket("embed"):
            return ops.embed(self.weight, tokens, scale=self.scale)


@register("embedding", "token_pair_embedding")
class TokenPairEmbedding(TokenEmbedding):
    """x[t] = E[token_t] * scale + P[(token_(t-1) * mul_prev + token_t * mul_cur) mod buckets], and P's last row (number
    `buckets`) for a sequence's first token.  The previous token is part of a sequence's state, so a prompt cut anywhere and
    one-token steps find it.  P: `params["pairs"]`, a full tensor name."""
    reads_step = True

    def __init__(self, params, prefix="model.embed_tokens."):
        super().__init__(params, prefix)
        self.buckets, self.mul_prev, self.mul_cur = int(params["buckets"]), int(params["mul_prev"]), int(params["mul_cur"])
        self.pairs_name = str(params["pairs"])
        if self.buckets < 1 or self.mul_prev < 0 or self.mul_cur < 0:
            raise ValueError("a pair table needs at least one bucket and multipliers that are not negative")

    def weights(self) -> List[WeightSpec]:
        return super().weights() + [WeightSpec(self.pairs_name, (self.buckets + 1, self.hidden))]

    def state_request(self) -> Optional[StateRequest]:
        return StateRequest((1,), torch.int32)

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        self.pairs = rt.place(tensors[self.pairs_name])
        if self.pairs.dtype != self.weight.dtype:
            self.pairs, self.weight = self.pairs.to(torch.float32), self.weight.to(torch.float32)

    def forward(self, step, memory) -> torch.Tensor:
        with ops.bucket("embed"):
            return ops.embed_pair(self.weight, self.pairs, step, memory.state, self.scale, self.mul_prev, self.mul_cur)


@register("head", "linear_head")
class LinearHead(Part):
    def __init__(self, params, prefix="lm_head."):
        super().__init__(params, prefix)
        self.vocab = int(params["vocab_size"])
        self.hidden = int(params["hidden_size"])
        self.tied = bool(params.get("tied", False))
        self.scale = float(params.get("scale", 1.0))        # logits = scale * (W h)
        self.softcap = float(params.get("softcap") or 0.0)  # > 0: logits = c tanh(logits / c)
        self.weight: Optional[torch.Tensor] = None

    def weights(self) -> List[WeightSpec]:
        return [] if self.tied else [WeightSpec(self.tensor_name("weight", "weight"), (self.vocab, self.hidden))]

    def ignorable(self) -> List[str]:
        """Names a file may carry without their being used (a tied model that still stores its head)."""
        return [self.tensor_name("weight", "weight")] if self.tied else []

    def bind(self, tensors, rt, embedding: Optional[TokenEmbedding] = None) -> None:
        super().bind(tensors, rt)
        if self.tied:
            if embedding is None:
                raise ValueError("a tied head needs the embedding it is tied to")
            self.weight = embedding.weight
        else:
            self.weight = rt.place(tensors[self.tensor_name("weight", "weight")])

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        with ops.bucket("logits"):
            logits = linear(h, self.weight, out_dtype=torch.float32)
            if self.scale != 1.0:
                logits = ops.scale_rows(logits, self.scale)
            return ops.softcap_rows(logits, self.softcap) if self.softcap > 0 else logits

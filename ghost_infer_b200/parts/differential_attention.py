"""Differential attention: every head is one map of attention less a share of another over the same values.

With h the mixer's input, H heads, G key/value heads (head a reads key/value head a / (H / G)), maps of `head_dim` numbers and
values of `v_head_dim`:

    q = Wq h (H x 2 maps x head_dim),  k = Wk h (G x 2 x head_dim),  v = Wv h (G x v_head_dim)
    `conv` taps > 0: each channel of q, k and v passes a causal convolution over the sequence's tokens, no bias, no activation,
               zeros before the start; the last tap is the token's own
    the first `rotary.dims` numbers of every map of q and k turn by the position's angles (pairs as `rotary.pairing` says)
    score = (q . k) * scale, map by map; position i sees j <= i, with `chunk` = s only those of its own chunk, floor(i / s) =
               floor(j / s); softmax in 32-bit gives a1 and a2
    lambda = exp(sum(lq1 lk1)) - exp(sum(lq2 lk2)) + diff
    o = a1 - lambda a2, divided by its root mean square over the head's values (eps), times 1 - diff
    residual += Wo (heads)

A cached key row is the two maps side by side, and a head's two queries are rows of that width with zeros in the other map's
place: grouped-query attention with 2 H queries over G key/value heads, in which one read of a key row and of a value serves both
maps of every head of the group.  Per sequence the convolution keeps its last `conv` - 1 inputs, float32.

Tensor names: prefix + `base` + {q, q.conv, k, k.conv, v, v.conv, lq1, lk1, lq2, lk2, o} (`base` "mix.").
"""
from __future__ import annotations

import math
from typing import List, Optional

import torch

from ..cache.sequence_cache import CacheRequest, StateRequest
from ..kernels import ops
from .base import Mixer, WeightSpec
from .linear import linear, stack_rows
from .registry import register
from .rope import Rotary

_KEYS = ("q", "q.conv", "k", "k.conv", "v", "v.conv", "lq1", "lk1", "lq2", "lk2", "o")


@register("mixer", "differential_attention")
class DifferentialAttention(Mixer):
    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden = int(params["hidden_size"])
        self.n_heads = int(params["num_heads"])
        self.n_kv = int(params["num_kv_heads"])
        self.head_dim = int(params["head_dim"])
        self.v_dim = int(params.get("v_head_dim") or self.head_dim)
        self.scale = float(params["scale"])
        self.diff = float(params["diff"])
        self.taps = int(params.get("conv") or 0)
        self.chunk = int(params["chunk"]) if params.get("chunk") else None
        self.eps = float(params.get("eps", 1e-6))
        if self.n_heads % self.n_kv:
            raise ValueError(f"{self.n_heads} heads do not divide into {self.n_kv} kv heads")
        rot = params.get("rotary")
        self.rotary, self.rot_dims = None, 0
        if rot is not None and int(rot["dims"]) > 0:
            self.rot_dims = int(rot["dims"])
            self.rotary = Rotary({"head_dim": self.head_dim, "rotary_dim": self.rot_dims, "theta": float(rot["base"]),
                                  "pairing": rot.get("pairing", "adjacent"), "scaling": rot.get("scaling")}, prefix)
        self.adjacent = self.rotary is not None and self.rotary.pairing == "adjacent"
        self.key_width = 2 * self.head_dim                     # a cached key row: both maps
        self.q_dim, self.k_dim, self.v_width = self.n_heads * self.key_width, self.n_kv * self.key_width, self.n_kv * self.v_dim
        self.channels = self.q_dim + self.k_dim + self.v_width
        base = str(params.get("base", "mix."))
        self.names = {k: self.tensor_name(k, base + k) for k in _KEYS}

    def weights(self) -> List[WeightSpec]:
        n, d = self.names, self.hidden
        out = [WeightSpec(n["q"], (self.q_dim, d)), WeightSpec(n["k"], (self.k_dim, d)), WeightSpec(n["v"], (self.v_width, d)),
               WeightSpec(n["o"], (d, self.n_heads * self.v_dim))]
        if self.taps:
            out += [WeightSpec(n["q.conv"], (self.q_dim, self.taps)), WeightSpec(n["k.conv"], (self.k_dim, self.taps)),
                    WeightSpec(n["v.conv"], (self.v_width, self.taps))]
        return out + [WeightSpec(n[k], (self.head_dim,)) for k in ("lq1", "lk1", "lq2", "lk2")]

    def cache_request(self) -> Optional[CacheRequest]:
        v = None if self.v_dim == self.key_width else self.v_dim
        if self.chunk:
            return CacheRequest("chunk", self.n_kv, self.key_width, self.chunk, v)
        return CacheRequest("full", self.n_kv, self.key_width, None, v)

    def state_request(self) -> Optional[StateRequest]:
        return StateRequest(((self.taps - 1) * self.channels,), torch.float32) if self.taps > 1 else None

    def decode_plan(self, n_seqs: int, max_kv_len: int, sm_count: int, kv_lens=None):
        return ops.attn_general_decode_plan(n_seqs, max_kv_len, sm_count, 2 * self.n_heads, self.n_kv, None, self.chunk, self.rt.dtype,
                                            self.key_width, self.v_dim, kv_lens)

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        n = self.names
        self.w_in = stack_rows([rt.place(tensors[n[k]]) for k in ("q", "k", "v")])
        self.w_o = rt.place(tensors[n["o"]])
        self.conv_w = None
        if self.taps:
            # [taps, channels]: a tap of neighbouring channels side by side, 32-bit
            self.conv_w = torch.cat([tensors[n[k]].to(torch.float32) for k in ("q.conv", "k.conv", "v.conv")], dim=0).t().to(rt.device).contiguous()
        vec = lambda k: tensors[n[k]].to(device="cpu", dtype=torch.float64)
        self.map_weight = math.exp(float(vec("lq1") @ vec("lk1"))) - math.exp(float(vec("lq2") @ vec("lk2"))) + self.diff
        if self.rotary is not None:
            self.rotary.bind(tensors, rt)

    def forward(self, h, residual, step, memory) -> None:
        if memory.k is None or not memory.writes:
            raise RuntimeError("differential attention was given no cache of its own")
        if self.taps > 1 and memory.state is None:
            raise RuntimeError("the convolution was given no per-sequence state")
        with ops.bucket("qkv matmul"):
            rows = linear(h, self.w_in, out_dtype=torch.float32)
        with ops.bucket("rope+cache"):
            table = self.rotary.table(step) if self.rotary is not None else None
            q = ops.map_prepare(rows, self.rt.dtype, self.conv_w, memory.state, table, self.rot_dims, self.adjacent, step, memory,
                                self.n_heads, self.n_kv, self.head_dim, self.v_dim)
        with ops.bucket("attention"):
            att = torch.empty((q.shape[0], 2 * self.n_heads * self.v_dim), dtype=self.rt.dtype, device=q.device)
            ops.attention_general(q, memory, step, 2 * self.n_heads, self.n_kv, self.key_width, self.v_dim, self.scale, att,
                                  chunk=self.chunk, plan=step.plan_of(self))
            att = ops.map_difference(att, self.n_heads, self.v_dim, self.map_weight, 1.0 - self.diff, self.eps)
        with ops.bucket("out matmul"):
            linear(att, self.w_o, out=residual, accumulate=True)

"""Causal attention whose keys and values come out of one low-rank latent per token ("latent attention").

With h the mixer's input, H heads, a head's query and key made of `dim` unrotated and `rot_dim` rotated numbers, values
of `v_dim` numbers, a latent of `rank` numbers and a query latent of `q_rank`:

    cq = rmsnorm(W_dq h) * w_dq_norm                      q = W_uq cq, per head [dim | rot_dim]   (no q_rank: q = W_q h)
    [a | kr] = W_dkv h   (rank | rot_dim numbers)         c = rmsnorm(a) * w_dkv_norm
    k_h = W_uk,h c       v_h = W_uv,h c                   kr: one rotated key part shared by all heads
    score_h(i, j) = (q_h,unrot(i) . k_h(j) + rot(q_h,rot(i)) . rot(kr(j))) * scale,   j <= i,   softmax,   out = W_o [sum p v_h]

The position encoding (`params["position"]`, a rotary part) turns the rotated parts only; values are not rotated; `scale`
is used as given.  Options: `window` w (i sees j with i - j < w; the cache keeps no more); `sink` (a learned number per head,
one more term exp(sink) of the softmax's denominator; tensor "sink"); `out_gate` "sigmoid": the heads side by side are
multiplied by sigmoid(W_g h) (tensor "g") before W_o, or "head_sigmoid": W_g h is one number per head.
Only c and the rotated kr are cached: one row [c | kr] per position, shared by all heads and serving
as key and as value (`CacheRequest(values_in_keys=True)`).  To attend over such rows a head's unrotated query is carried
onto the latent, qa_h = W_uk,h^T q_h,unrot (so that qa_h . c = q_h,unrot . k_h), the attention runs with every head
reading the same rows, its result per head is a weighted sum of latents, and W_uv,h turns that into the head's values (which
is why one gate per head may as well multiply the sum of latents).
Norms, angles, scores and softmax are 32-bit.

Tensor names: prefix + "mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o}" ("mix.q" in place of the first three without a query latent;
"mix.g", "mix.sink") unless `params["tensor_names"]` gives others for the keys
"dq", "dq_norm", "uq", "q", "dkv", "dkv_norm", "uk", "uv", "o", "g", "sink".
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..cache.sequence_cache import CacheRequest
from ..kernels import ops
from .base import Mixer, WeightSpec
from .linear import linear, stack_rows
from .registry import lookup, register

_DEFAULT_NAMES = {"dq": "mix.dq", "dq_norm": "mix.dq.norm", "uq": "mix.uq", "dkv": "mix.dkv", "dkv_norm": "mix.dkv.norm",
                  "uk": "mix.uk", "uv": "mix.uv", "o": "mix.o", "g": "mix.g", "q": "mix.q", "sink": "mix.sink"}


@register("mixer", "latent_attention")
class LatentAttention(Mixer):
    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden = int(params["hidden_size"])
        self.n_heads = int(params["num_heads"])
        self.dim = int(params["head_dim"])              # unrotated numbers of a head's query and key
        self.rot_dim = int(params["rot_dim"])           # rotated numbers (the shared key part's width)
        self.v_dim = int(params["v_head_dim"])
        self.rank = int(params["kv_rank"])
        self.q_rank = int(params.get("q_rank") or 0)    # 0: queries straight from the input
        self.scale = float(params["scale"])
        self.eps = float(params["eps"])
        self.out_gate = params.get("out_gate")
        if self.out_gate not in (None, "sigmoid", "head_sigmoid"):
            raise ValueError(f"out_gate must be None, \"sigmoid\" or \"head_sigmoid\", got {self.out_gate!r}")
        self.window = int(params["window"]) if params.get("window") else None
        self.sink = bool(params.get("sink", False))
        if min(self.n_heads, self.dim, self.v_dim, self.rank) < 1 or self.rot_dim < 0 or self.q_rank < 0:
            raise ValueError("latent attention: sizes must be positive")
        pos = params.get("position")
        self.position = lookup("position", pos.kind)(pos.params, prefix) if pos is not None and self.rot_dim > 0 else None
        self.rot = int(self.position.rotary_dim) if self.position is not None else 0     # how many of rot_dim turn
        if self.rot > self.rot_dim:
            raise ValueError(f"latent attention: {self.rot} numbers cannot turn in a rotated part of {self.rot_dim}")
        if self.position is not None and getattr(self.position, "pairing", "adjacent") != "adjacent":
            raise ValueError("latent attention turns neighbouring pairs: the position encoding must pair (2i, 2i + 1)")
        self.names = {k: self.tensor_name(k, v) for k, v in _DEFAULT_NAMES.items()}

    def weights(self) -> List[WeightSpec]:
        n, H = self.names, self.n_heads
        out = []
        if self.out_gate:
            out.append(WeightSpec(n["g"], (H if self.out_gate == "head_sigmoid" else H * self.v_dim, self.hidden)))
        if self.sink:
            out.append(WeightSpec(n["sink"], (H,)))
        qd = H * (self.dim + self.rot_dim)
        if self.q_rank:
            out += [WeightSpec(n["dq"], (self.q_rank, self.hidden)), WeightSpec(n["dq_norm"], (self.q_rank,), "ones"),
                    WeightSpec(n["uq"], (qd, self.q_rank))]
        else:
            out.append(WeightSpec(n["q"], (qd, self.hidden)))
        return out + [WeightSpec(n["dkv"], (self.rank + self.rot_dim, self.hidden)), WeightSpec(n["dkv_norm"], (self.rank,), "ones"),
                WeightSpec(n["uk"], (H * self.dim, self.rank)), WeightSpec(n["uv"], (H * self.v_dim, self.rank)),
                WeightSpec(n["o"], (self.hidden, H * self.v_dim))]

    def cache_request(self) -> Optional[CacheRequest]:
        return CacheRequest("window" if self.window else "full", 1, self.rank + self.rot_dim, self.window, self.rank, values_in_keys=True)

    def decode_plan(self, n_seqs: int, max_kv_len: int, sm_count: int, kv_lens=None):
        return ops.attn_latent_decode_plan(n_seqs, max_kv_len, sm_count, self.n_heads, self.rank, self.rot_dim, self.rt.dtype,
                                           self.window)

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        n, H = self.names, self.n_heads
        place = lambda key: rt.place(tensors[n[key]])
        per_head = self.out_gate == "head_sigmoid"
        if self.q_rank:
            dq, dkv = place("dq"), place("dkv")
            if dq.dtype != dkv.dtype:
                dq, dkv = dq.to(torch.float32), dkv.to(torch.float32)
            self.w_down = torch.cat([dq, dkv], dim=0).contiguous()   # one product: [query latent | latent | rotary key part]
            self.w_uq = place("uq")
        else:
            # one product: [latent | rotary key part | queries | heads' gates]
            self.w_down = stack_rows([place(k) for k in (("dkv", "q", "g") if per_head else ("dkv", "q"))])
        self.w_g = place("g") if (self.out_gate and not (per_head and not self.q_rank)) else None
        self.w_o = place("o")
        self.sinks = tensors[n["sink"]].to(device=rt.device, dtype=torch.float32).contiguous() if self.sink else None
        # per head: W_uk,h^T as [rank, dim] (rows of the carried query), W_uv,h as [v_dim, rank]
        self.w_uk_t = place("uk").view(H, self.dim, self.rank).transpose(1, 2).contiguous()
        self.w_uv = place("uv").view(H, self.v_dim, self.rank).contiguous()
        qn, cn = place("dq_norm") if self.q_rank else None, place("dkv_norm")
        if qn is not None and qn.dtype != cn.dtype:
            qn, cn = qn.to(torch.float32), cn.to(torch.float32)
        self.w_q_norm, self.w_c_norm = qn, cn
        if self.position is not None:
            self.position.bind(tensors, rt)

    def forward(self, h, residual, step, memory) -> None:
        H, T, dt = self.n_heads, h.shape[0], self.rt.dtype
        with ops.bucket("qkv matmul"):
            down = linear(h, self.w_down, out_dtype=dt)
            qa = torch.empty((T, H * (self.rank + self.rot_dim)), dtype=dt, device=h.device)
        with ops.bucket("rope+cache"):
            table = self.position.table(step) if self.position is not None else None
            where = (step.positions, step.token_slots, memory, self.q_rank, self.rank, self.rot_dim)
            own = self.q_rank + self.rank + self.rot_dim
            if self.q_rank:
                cq = ops.latent_prepare(down, self.w_q_norm, self.w_c_norm, self.eps, table, self.rot, *where)
            else:
                q = down[:, own:own + H * (self.dim + self.rot_dim)]
                ops.latent_prepare(down[:, :own], None, self.w_c_norm, self.eps, table, self.rot, *where, queries=(qa, q, H, self.dim))
        with ops.bucket("qkv matmul"):
            if self.q_rank:
                q = linear(cq, self.w_uq, out_dtype=dt)
            ops.bmm_heads(qa, self.rank + self.rot_dim, q, self.dim + self.rot_dim, self.w_uk_t, self.rank, self.dim)
        if self.q_rank:
            with ops.bucket("rope+cache"):
                ops.latent_query_rot(qa, q, table, self.rot, H, self.dim, self.rot_dim, self.rank)
        gate = None
        if self.out_gate == "head_sigmoid":
            if self.w_g is not None:
                with ops.bucket("out matmul"):
                    gate = linear(h, self.w_g, out_dtype=dt)
            else:
                at = own + H * (self.dim + self.rot_dim)
                gate = down[:, at:at + H]
        with ops.bucket("attention"):
            lat = torch.empty((T, H * self.rank), dtype=dt, device=h.device)
            lat = ops.attention_latent(qa, memory, step, H, self.rank, self.rot_dim, self.scale, lat, plan=step.plan_of(self),
                                       window=self.window, sinks=self.sinks, gate=gate)
        with ops.bucket("out matmul"):
            att = torch.empty((T, H * self.v_dim), dtype=dt, device=h.device)
            ops.bmm_heads(att, self.v_dim, lat, self.rank, self.w_uv, self.v_dim, self.rank)
            if self.out_gate == "sigmoid":
                att = ops.gate_mul(att, linear(h, self.w_g, out_dtype=dt), "sigmoid")
            linear(att, self.w_o, out=residual, accumulate=True)

"""Mixers that carry a matrix of state per head from token to token: a gated delta rule, decayed linear attention, retention, gated
linear attention.

All walk, per head, S (a key_dim x v_dim matrix of 32-bit numbers, zero when a sequence starts):

    S <- g_t S;   u_t = v_t (or, delta rule: beta_t (v_t - S^T k_t));   S <- S + k_t u_t^T;   o_t = S^T q_t

"gated_delta_rule": q = Wq h and k = Wk h (`qk_heads` heads of key_dim; head a reads query/key head a / (heads / qk_heads)),
v = Wv h (heads of v_dim); each passes a causal convolution over `conv` tokens per channel (no bias; the last tap is the
current token's; zeros before the start) and silu; q and k become unit vectors per head, x / sqrt(sum x^2 + `unit_eps`), q
also times key_dim^(-1/2); beta = sigmoid(Wb h) and g = exp(-exp(A_log) softplus(Wa h + dt_bias)), one per head.  Each
head's o is divided by its root mean square over v_dim (eps), times a weight of v_dim shared by the heads, times
silu(Wg h); residual += Wo (...).  Per sequence: S and the convolution's last `conv` - 1 inputs, one float32 row.

"decayed_linear_attention": q, k = silu(Wq h), silu(Wk h) (heads of key_dim), v = silu(Wv h) (heads of v_dim); g is a
constant per head (`decay`); the concatenated heads are RMS-normed together (weight of heads * v_dim, eps), multiplied by
sigmoid(Wg h), and projected: residual += Wo (...).  Per sequence: S.

"retention": q = Wq h, k = Wk h (heads of key_dim), v = Wv h (heads of v_dim), no activation; the position encoding
(`params["position"]`, a rotary part, or None) turns q and k, and k is multiplied by key_dim^(-1/2); g is a constant per head
(`decay`); each head's o is divided by its root mean square over v_dim (eps, no weight), the heads side by side are multiplied
by silu(Wg h), and projected: residual += Wo (...).  Per sequence: S.

"gated_linear_attention": q = Wq h, times key_dim^(-1/2), and k = Wk h (heads of key_dim), v = Wv h (heads of v_dim), no
activation; the decay is one number per key channel and token, S <- diag(g_t) S, g = sigmoid(Wa2 (Wa1 h) + b)^(1 / `tau`)
(heads * key_dim of them; the width between Wa1 and Wa2 is the tensors'); each head's o is divided by its root mean square over
v_dim (eps), times a weight of v_dim shared by the heads, times silu(Wg h), and projected: residual += Wo (...).  Per sequence: S.

The recurrence, decays, gates of the recurrence, unit norms and output norms are 32-bit in both precisions.
Tensor names: prefix + `base` + {q, q.conv, k, k.conv, v, v.conv, b, a, A_log, dt_bias, a1, a2, a2.b, norm, g, o} (`base` "mix.").
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..cache.sequence_cache import StateRequest
from ..kernels import ops
from .base import Mixer, WeightSpec
from .linear import linear, stack_rows
from .registry import lookup, register


@register("mixer", "gated_delta_rule")
class GatedDeltaRule(Mixer):
    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["heads"])
        self.qk_heads = int(params["qk_heads"])
        self.key_dim = int(params["key_dim"])
        self.v_dim = int(params["v_dim"])
        self.taps = int(params["conv"])
        self.eps = float(params["eps"])
        self.unit_eps = float(params.get("unit_eps", 1e-6))
        if self.heads % self.qk_heads:
            raise ValueError(f"{self.heads} heads do not divide into {self.qk_heads} query/key heads")
        if self.taps < 1:
            raise ValueError("the convolution needs at least one tap")
        self.qk_width, self.v_width = self.qk_heads * self.key_dim, self.heads * self.v_dim
        self.channels = 2 * self.qk_width + self.v_width
        self.s_floats = self.heads * self.key_dim * self.v_dim
        base = str(params.get("base", "mix."))
        keys = ("q", "q.conv", "k", "k.conv", "v", "v.conv", "b", "a", "A_log", "dt_bias", "norm", "g", "o")
        self.names = {k: self.tensor_name(k, base + k) for k in keys}

    def weights(self) -> List[WeightSpec]:
        n, d = self.names, self.hidden
        return [WeightSpec(n["q"], (self.qk_width, d)), WeightSpec(n["q.conv"], (self.qk_width, self.taps)),
                WeightSpec(n["k"], (self.qk_width, d)), WeightSpec(n["k.conv"], (self.qk_width, self.taps)),
                WeightSpec(n["v"], (self.v_width, d)), WeightSpec(n["v.conv"], (self.v_width, self.taps)),
                WeightSpec(n["b"], (self.heads, d)), WeightSpec(n["A_log"], (self.heads,)),
                WeightSpec(n["norm"], (self.v_dim,), "ones"), WeightSpec(n["a"], (self.heads, d)),
                WeightSpec(n["dt_bias"], (self.heads,)), WeightSpec(n["g"], (self.v_width, d)),
                WeightSpec(n["o"], (d, self.v_width))]

    def state_request(self) -> Optional[StateRequest]:
        return StateRequest((self.s_floats + (self.taps - 1) * self.channels,), torch.float32)

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        n = self.names
        # one product: [q | k | v | gate | beta | decay]; the convolved channels come first
        self.w_in = stack_rows([rt.place(tensors[n[k]]) for k in ("q", "k", "v", "g", "b", "a")])
        self.w_o = rt.place(tensors[n["o"]])
        cw = [rt.place(tensors[n[k]]) for k in ("q.conv", "k.conv", "v.conv")]
        if len({c.dtype for c in cw}) > 1:
            cw = [c.to(torch.float32) for c in cw]
        self.conv_w = torch.cat(cw, dim=0).contiguous()
        self.conv_b = torch.zeros((self.channels,), dtype=self.conv_w.dtype, device=rt.device)     # the design has no bias
        # the recurrence's constants and the norm's weight enter 32-bit arithmetic: kept as 32-bit values
        f32 = lambda name: tensors[name].to(device=rt.device, dtype=torch.float32).contiguous()
        self.a_log, self.dt_bias, self.norm_w = f32(n["A_log"]), f32(n["dt_bias"]), f32(n["norm"])

    def forward(self, h, residual, step, memory) -> None:
        if memory.state is None:
            raise RuntimeError("the delta rule was given no per-sequence state")
        C, qk, vw, H = self.channels, self.qk_width, self.v_width, self.heads
        with ops.bucket("qkv matmul"):
            proj = linear(h, self.w_in, out_dtype=self.rt.dtype)
        with ops.bucket("conv"):
            conv = ops.mamba2_conv(proj, self.conv_w, self.conv_b, memory.state, step, 0, C, self.taps, self.s_floats)
        with ops.bucket("scan"):
            o = ops.linear_state(conv[:, :qk], conv[:, qk:2 * qk], conv[:, 2 * qk:], memory.state, step, H, self.qk_heads,
                                 self.key_dim, self.v_dim, self.a_log, decay_in=proj[:, C + vw + H:C + vw + 2 * H],
                                 dt_bias=self.dt_bias, beta_in=proj[:, C + vw:C + vw + H], unit_norm=True,
                                 norm_eps=self.unit_eps, q_scale=self.key_dim ** -0.5, delta=True)
        with ops.bucket("gated norm"):
            y = ops.norm_gate(o, proj[:, C:C + vw], self.norm_w, self.v_dim, self.eps, "silu", self.rt.dtype)
        with ops.bucket("out matmul"):
            linear(y, self.w_o, out=residual, accumulate=True)


@register("mixer", "decayed_linear_attention")
class DecayedLinearAttention(Mixer):
    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["heads"])
        self.key_dim = int(params["key_dim"])
        self.v_dim = int(params["v_dim"])
        self.eps = float(params["eps"])
        self.decay = tuple(float(g) for g in params["decay"])
        if len(self.decay) != self.heads:
            raise ValueError(f"{len(self.decay)} decays for {self.heads} heads")
        self.qk_width, self.v_width = self.heads * self.key_dim, self.heads * self.v_dim
        base = str(params.get("base", "mix."))
        self.names = {k: self.tensor_name(k, base + k) for k in ("q", "k", "v", "g", "o", "norm")}

    def weights(self) -> List[WeightSpec]:
        n, d = self.names, self.hidden
        return [WeightSpec(n["q"], (self.qk_width, d)), WeightSpec(n["k"], (self.qk_width, d)), WeightSpec(n["v"], (self.v_width, d)),
                WeightSpec(n["g"], (self.v_width, d)), WeightSpec(n["o"], (d, self.v_width)),
                WeightSpec(n["norm"], (self.v_width,), "ones")]

    def state_request(self) -> Optional[StateRequest]:
        return StateRequest((self.heads * self.key_dim * self.v_dim,), torch.float32)

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        n = self.names
        self.w_in = stack_rows([rt.place(tensors[n[k]]) for k in ("q", "k", "v", "g")])
        self.w_o = rt.place(tensors[n["o"]])
        self.norm_w = tensors[n["norm"]].to(device=rt.device, dtype=torch.float32).contiguous()
        self.decay_dev = torch.tensor(self.decay, dtype=torch.float64).to(device=rt.device, dtype=torch.float32)

    def forward(self, h, residual, step, memory) -> None:
        if memory.state is None:
            raise RuntimeError("linear attention was given no per-sequence state")
        qk, vw = self.qk_width, self.v_width
        with ops.bucket("qkv matmul"):
            proj = linear(h, self.w_in, out_dtype=self.rt.dtype)
        with ops.bucket("scan"):
            o = ops.linear_state(proj[:, :qk], proj[:, qk:2 * qk], proj[:, 2 * qk:2 * qk + vw], memory.state, step, self.heads,
                                 self.heads, self.key_dim, self.v_dim, self.decay_dev, in_act=True)
        with ops.bucket("gated norm"):
            y = ops.norm_gate(o, proj[:, 2 * qk + vw:2 * qk + 2 * vw], self.norm_w, vw, self.eps, "sigmoid", self.rt.dtype)
        with ops.bucket("out matmul"):
            linear(y, self.w_o, out=residual, accumulate=True)


@register("mixer", "retention")
class Retention(Mixer):
    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["heads"])
        self.key_dim = int(params["key_dim"])
        self.v_dim = int(params["v_dim"])
        self.eps = float(params["eps"])
        self.decay = tuple(float(g) for g in params["decay"])
        if len(self.decay) != self.heads:
            raise ValueError(f"{len(self.decay)} decays for {self.heads} heads")
        pos = params.get("position")
        self.position = lookup("position", pos.kind)(pos.params, prefix) if pos is not None else None
        self.rot = int(self.position.rotary_dim) if self.position is not None else 0
        self.adjacent = self.position is not None and self.position.pairing == "adjacent"
        self.qk_width, self.v_width = self.heads * self.key_dim, self.heads * self.v_dim
        base = str(params.get("base", "mix."))
        self.names = {k: self.tensor_name(k, base + k) for k in ("q", "k", "v", "g", "o")}

    def weights(self) -> List[WeightSpec]:
        n, d = self.names, self.hidden
        return [WeightSpec(n["q"], (self.qk_width, d)), WeightSpec(n["k"], (self.qk_width, d)), WeightSpec(n["v"], (self.v_width, d)),
                WeightSpec(n["g"], (self.v_width, d)), WeightSpec(n["o"], (d, self.v_width))]

    def state_request(self) -> Optional[StateRequest]:
        return StateRequest((self.heads * self.key_dim * self.v_dim,), torch.float32)

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        n = self.names
        self.w_in = stack_rows([rt.place(tensors[n[k]]) for k in ("q", "k", "v", "g")])
        self.w_o = rt.place(tensors[n["o"]])
        self.decay_dev = torch.tensor(self.decay, dtype=torch.float64).to(device=rt.device, dtype=torch.float32)
        if self.position is not None:
            self.position.bind(tensors, rt)

    def forward(self, h, residual, step, memory) -> None:
        if memory.state is None:
            raise RuntimeError("retention was given no per-sequence state")
        qk, vw = self.qk_width, self.v_width
        with ops.bucket("qkv matmul"):
            proj = linear(h, self.w_in, out_dtype=self.rt.dtype)
        with ops.bucket("scan"):
            table = self.position.table(step) if self.position is not None else None
            o = ops.linear_state_rot(proj[:, :qk], proj[:, qk:2 * qk], proj[:, 2 * qk:2 * qk + vw], memory.state, step, self.heads,
                                     self.key_dim, self.v_dim, self.decay_dev, table, self.rot, self.adjacent, self.key_dim ** -0.5)
        with ops.bucket("gated norm"):
            y = ops.norm_gate(o, proj[:, 2 * qk + vw:2 * qk + 2 * vw], None, self.v_dim, self.eps, "silu", self.rt.dtype)
        with ops.bucket("out matmul"):
            linear(y, self.w_o, out=residual, accumulate=True)


@register("mixer", "gated_linear_attention")
class GatedLinearAttention(Mixer):
    RANK = 16          # the width between the decay's two matrices where no file says another (random weights)

    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden = int(params["hidden_size"])
        self.heads = int(params["heads"])
        self.key_dim = int(params["key_dim"])
        self.v_dim = int(params["v_dim"])
        self.tau = float(params["tau"])
        self.eps = float(params["eps"])
        self.rank = int(params.get("rank") or self.RANK)
        if not self.tau > 0:
            raise ValueError(f"the decays' root must be positive, got {self.tau}")
        self.qk_width, self.v_width = self.heads * self.key_dim, self.heads * self.v_dim
        base = str(params.get("base", "mix."))
        self.names = {k: self.tensor_name(k, base + k) for k in ("q", "k", "v", "g", "o", "norm", "a1", "a2", "a2.b")}

    def weights(self) -> List[WeightSpec]:
        n, d = self.names, self.hidden
        return [WeightSpec(n["q"], (self.qk_width, d)), WeightSpec(n["k"], (self.qk_width, d)), WeightSpec(n["v"], (self.v_width, d)),
                WeightSpec(n["g"], (self.v_width, d)), WeightSpec(n["o"], (d, self.v_width)), WeightSpec(n["norm"], (self.v_dim,), "ones"),
                WeightSpec(n["a1"], (self.rank, d), free=(0,)), WeightSpec(n["a2"], (self.qk_width, self.rank), free=(1,)),
                WeightSpec(n["a2.b"], (self.qk_width,))]

    def state_request(self) -> Optional[StateRequest]:
        return StateRequest((self.heads * self.key_dim * self.v_dim,), torch.float32)

    def bind(self, tensors, rt) -> None:
        super().bind(tensors, rt)
        n = self.names
        a1, a2 = tensors[n["a1"]], tensors[n["a2"]]
        self.rank = int(a1.shape[0])
        if int(a2.shape[1]) != self.rank:
            raise ValueError(f"{n['a1']} has {self.rank} rows, {n['a2']} takes {int(a2.shape[1])}")
        # one product: [q | k | v | gate | what the decays are made of]
        self.w_in = stack_rows([rt.place(tensors[n[k]]) for k in ("q", "k", "v", "g", "a1")])
        self.w_o = rt.place(tensors[n["o"]])
        # what makes the decays and the norm enters 32-bit arithmetic: kept as 32-bit values (a2 with its outputs side by side)
        f32 = lambda t: t.to(device=rt.device, dtype=torch.float32).contiguous()
        self.a2_t, self.a2_b, self.norm_w = f32(a2.to(torch.float32).t()), f32(tensors[n["a2.b"]]), f32(tensors[n["norm"]])

    def forward(self, h, residual, step, memory) -> None:
        if memory.state is None:
            raise RuntimeError("linear attention was given no per-sequence state")
        qk, vw = self.qk_width, self.v_width
        g0 = 2 * qk + vw
        with ops.bucket("qkv matmul"):
            proj = linear(h, self.w_in, out_dtype=self.rt.dtype)
        with ops.bucket("scan"):
            keep = ops.key_decays(proj[:, g0 + vw:g0 + vw + self.rank], self.a2_t, self.a2_b, self.tau)
            o = ops.linear_state_keyed(proj[:, :qk], proj[:, qk:2 * qk], proj[:, 2 * qk:g0], keep, memory.state, step, self.heads,
                                       self.key_dim, self.v_dim, self.key_dim ** -0.5)
        with ops.bucket("gated norm"):
            y = ops.norm_gate(o, proj[:, g0:g0 + vw], self.norm_w, self.v_dim, self.eps, "silu", self.rt.dtype)
        with ops.bucket("out matmul"):
            linear(y, self.w_o, out=residual, accumulate=True)

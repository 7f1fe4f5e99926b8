"""Arrangements of a layer's parts around the residual stream."""
from __future__ import annotations

import torch

from ..kernels import ops
from .base import Block
from .registry import register


@register("block", "prenorm_residual")
class PreNormResidual(Block):
    """x += mixer(norm(x)); x += ffn(norm(x)), the residual stream x kept in 32-bit
    (src/model.rs:996-1147; the reference's stream is f32 too, src/model.rs:704-705)."""

    def first_reader(self):
        return self.mixer_norm

    def forward(self, x, step, memory) -> None:
        # The last product of the mixer and of the feed-forward adds into x; in a decode step it may leave
        # partial sums pending for the norm that reads x next (a norm that cannot add them has them settled first).
        if x.is_cuda and not getattr(self.mixer_norm, "settles_pending", False):
            ops.settle(x)
        h = self.mixer_norm.forward(x)
        with ops.defer_into(x):
            self.mixer.forward(h, x, step, memory)
        if self.ffn is None:          # a layer without a feed-forward: the mixer alone
            return
        if x.is_cuda and not getattr(self.ffn_norm, "settles_pending", False):
            ops.settle(x)
        h = self.ffn_norm.forward(x)
        with ops.defer_into(x):
            self.ffn.forward(h, x, step)


@register("block", "residual_postnorm")
class ResidualPostNorm(Block):
    """x += s1 * norm(mixer(x)); x += s2 * norm(ffn(x)): the sublayers read the stream itself (in the activation type)
    and the norm sits on what they give back; s1 and s2 are learned per-channel scales (`extra["mixer_scale"]`,
    `extra["ffn_scale"]`, each optional).  Then every `extra` part named "after..." runs in order as a feed-forward
    on the stream (it adds to it by itself).  Norms, scales and sums are 32-bit."""

    def forward(self, x, step, memory) -> None:
        if x.is_cuda:
            ops.settle(x)             # nothing here defers into the stream; what a layer before left is added first
        dt = self.mixer_norm.rt.dtype
        low = dt != torch.float32     # the 32-bit path reads the stream itself
        subs = [(self.mixer_norm, self.extra.get("mixer_scale"), lambda h, y: self.mixer.forward(h, y, step, memory))]
        if self.ffn is not None:
            subs.append((self.ffn_norm, self.extra.get("ffn_scale"), lambda h, y: self.ffn.forward(h, y, step)))
        after = [part for name, part in self.extra.items() if name.startswith("after")]
        # one matrix of 32-bit rows that every sublayer adds into, and one copy of the stream in the activation type: the
        # pass that joins a sublayer's output to the stream zeroes the first and renews the second for the next reader
        y = torch.empty(x.shape, dtype=torch.float32, device=x.device)
        h = ops.cast_rows(x, dt, zero=y)
        for i, (norm, scale, run) in enumerate(subs):
            run(h, y)
            more, reader = i + 1 < len(subs), i + 1 < len(subs) or bool(after)
            norm.add_normed(x, y, scale.weight if scale is not None else None, cast_out=h if (low and reader) else None, zero_y=more)
        for i, part in enumerate(after):
            part.forward(h, x, step)
            if low and i + 1 < len(after):
                h = ops.cast_rows(x, dt)


@register("block", "sandwich_residual")
class SandwichResidual(Block):
    """x += n1b(mixer(n1(x))); x += n2b(ffn(n2(x))): a norm before every sublayer and one on what it gives back
    (`extra["mixer_post"]`, `extra["ffn_post"]`).  Stream, norms and sums are 32-bit.  A sublayer's last product may leave partial
    sums pending in its rows; a norm whose `join` can do so adds them, joins the rows to the stream and does the first operation
    of whoever reads the stream next, in one pass; other norms do these one after the other."""

    def first_reader(self):
        return self.mixer_norm

    def _sublayer(self, x, step, pre, post, run, reader) -> None:
        if x.is_cuda and not getattr(pre, "settles_pending", False):
            ops.settle(x)
        h = pre.forward(x)
        # the rows a sublayer adds into: zeroed once a step, and again by every join for the next sublayer
        key = ("sublayer rows", tuple(x.shape))
        y = step.shared.get(key)
        if y is None:
            y = step.shared[key] = ops.as_carrier(torch.zeros(x.shape, dtype=torch.float32, device=x.device))
        with ops.defer_into(y):
            run(h, y)
        if hasattr(post, "join"):
            post.join(x, y, reader, step, zero_y=True)
        else:
            ops.settle(y)
            post.add_normed(x, y, zero_y=True)

    def forward(self, x, step, memory) -> None:
        last = step.next_reader
        self._sublayer(x, step, self.mixer_norm, self.extra["mixer_post"], lambda h, y: self.mixer.forward(h, y, step, memory),
                       self.ffn_norm if self.ffn is not None else last)
        if self.ffn is not None:
            self._sublayer(x, step, self.ffn_norm, self.extra["ffn_post"], lambda h, y: self.ffn.forward(h, y, step), last)


@register("block", "parallel_residual")
class ParallelResidual(Block):
    """x += s * (mixer(n(x)) + ffn(n(x))), s = `params["scale"]` (1 unless given): one norm, which both sublayers read.  They add
    into 32-bit rows of their own; one pass joins those to the stream (with whatever partial sums the two last products left in them),
    zeroes them for the next layer and, where the next reader of the stream is a norm that says so (`row_read`), does that norm
    on the way.  Stream, norms and sums are 32-bit."""

    def first_reader(self):
        return self.mixer_norm

    def forward(self, x, step, memory) -> None:
        if x.is_cuda and not getattr(self.mixer_norm, "settles_pending", False):
            ops.settle(x)
        h = self.mixer_norm.forward(x)
        key = ("sublayer rows", tuple(x.shape))
        y = step.shared.get(key)
        if y is None:
            y = step.shared[key] = ops.as_carrier(torch.zeros(x.shape, dtype=torch.float32, device=x.device))
        runs = [lambda: self.mixer.forward(h, y, step, memory)] if self.mixer is not None else []
        if self.ffn is not None:
            runs.append(lambda: self.ffn.forward(h, y, step))
        with ops.defer_into(y, two=True):      # nothing but the join reads the rows: both last products may leave it their sums
            for run in runs:
                run()
        reader = step.next_reader
        read = reader.row_read(step) if reader is not None and hasattr(reader, "row_read") else None
        with ops.bucket("norm"):
            nxt = ops.join_rows(x, y, float(self.params.get("scale", 1.0)), read)
        if nxt is not None:
            ops.hand_on(x, reader, nxt)

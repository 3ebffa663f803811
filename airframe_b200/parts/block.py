"""Arrangements of a layer's parts around the float32 residual stream.

``sandwich``: x += post(mixer(pre(x))); x += post(ff(pre(x))) - norms before
and after both halves; a layer whose feed-forward is of the kind ``none`` has
the first half only (reference order
``src/backend/bindless/pipeline/inference.rs:1096-1251``, net effect
x + norm(a) of ``sh_layer_v1.wgsl:834-849,869-884``).
``prenorm``: x += mixer(pre(x)); x += ff(pre(x)); a layer whose feed-forward
is of the kind ``none`` has the first half only.  Each residual sum is one
kernel with the norm that follows it (the feed-forward's, or the next layer's
first).
``postnorm``: x += post(mixer(x)); x += post(ff(x)): the sublayers read the
stream itself and the only norms stand behind them (each on the sublayer's output,
not on the sum); a layer whose feed-forward is of the kind ``none`` has the first
half only.  On the 16-bit path the kernel of a residual sum also writes the new
stream in 16 bits for the sublayer that reads it next.  A third sublayer of the
feed-forward kind (``side``) may follow, with its own norm behind it.
``normed_sum``: x <- norm1(alpha x + mixer(x)); x <- norm2(alpha x + ff(x)): the norm is
taken of the residual sum, so the stream itself is a norm's output; the sublayers read it as it stands.
Each sublayer's result may be multiplied element by element by sigmoid(W x + b) first, and what the
mixer reads may be shifted towards the token before, x_t + (x_(t-1) - x_t) * mu, whose row
is then part of a sequence's state, one for every run of the layer.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..config.base import ConfigError, PartSpec
from ..weights.loader import WeightDecl
from .base import Block, StateNeed, build_part, register_part
from .linear import PartialSums, as_terms, linear_split
from .norm import LayerNorm


@register_part("block", "sandwich")
class SandwichBlock(Block):
    roles = ("pre_mixer", "post_mixer", "pre_feed_forward", "post_feed_forward")

    def __init__(self, params, ctx, mixer, feed_forward, norms):
        if not feed_forward.present:
            self.roles = ("pre_mixer", "post_mixer")
        super().__init__(params, ctx, mixer, feed_forward, norms)

    def forward(self, x, batch, view, normed=None, next_pre=None):
        """Updates x in place.  ``normed`` may carry pre_mixer(x) made by the
        previous layer's last kernel; ``next_pre`` is the next layer's first
        norm, whose output is then returned (made by this layer's last kernel)."""
        n = self.norms
        dt = self.ctx.compute_dtype
        h = normed if normed is not None else n["pre_mixer"].forward(x, dt)
        a = self.mixer.forward(h, batch, view)
        if not self.feed_forward.present:
            return n["post_mixer"].add_normed(x, a, then=next_pre, out_dtype=dt)
        h = n["post_mixer"].add_normed(x, a, then=n["pre_feed_forward"], out_dtype=dt)
        f = self.feed_forward.forward(h, batch)
        return n["post_feed_forward"].add_normed(x, f, then=next_pre, out_dtype=dt)

    def first_norm(self):
        return self.norms["pre_mixer"]


@register_part("block", "prenorm")
class PreNormBlock(Block):
    roles = ("pre_mixer", "pre_feed_forward")

    def __init__(self, params, ctx, mixer, feed_forward, norms):
        if not feed_forward.present:
            self.roles = ("pre_mixer",)
        super().__init__(params, ctx, mixer, feed_forward, norms)

    def _add(self, x, a, then, dt):
        """x += a; returns then(x) when a norm follows."""
        if then is not None:
            return then.after_add(x, a, dt)
        kernels.add_scaled_rmsnorm(x, as_terms(a))
        return None

    def forward(self, x, batch, view, normed=None, next_pre=None):
        n = self.norms
        dt = self.ctx.compute_dtype
        h = normed if normed is not None else n["pre_mixer"].forward(x, dt)
        a = self.mixer.forward(h, batch, view)
        if not self.feed_forward.present:
            return self._add(x, a, next_pre, dt)
        h = self._add(x, a, n["pre_feed_forward"], dt)
        return self._add(x, self.feed_forward.forward(h, batch), next_pre, dt)

    def first_norm(self):
        return self.norms["pre_mixer"]


@register_part("block", "postnorm")
class PostNormBlock(Block):
    """Optional parameter ``side``: a PartSpec of category ``feed_forward``, run last (norm role ``post_side``)."""
    roles = ("post_mixer", "post_feed_forward")

    def __init__(self, params, ctx, mixer, feed_forward, norms):
        side = params.get("side")
        self.roles = ("post_mixer", *(("post_feed_forward",) if feed_forward.present else ()),
                      *(("post_side",) if side is not None else ()))
        super().__init__(params, ctx, mixer, feed_forward, norms)
        self.side = build_part("feed_forward", side, ctx) if side is not None else None
        # "the norm in front of a sublayer" is none: the stream as it stands, in the compute dtype
        self.reader = build_part("norm", PartSpec("as_is", {"size": norms["post_mixer"].size}), ctx)

    def children(self):
        return [*super().children(), *([self.side] if self.side is not None else [])]

    def forward(self, x, batch, view, normed=None, next_pre=None):
        dt = self.ctx.compute_dtype
        h = normed if normed is not None else self.reader.forward(x, dt)
        run = [("post_mixer", lambda h: self.mixer.forward(h, batch, view))]
        if self.feed_forward.present:
            run.append(("post_feed_forward", lambda h: self.feed_forward.forward(h, batch)))
        if self.side is not None:
            run.append(("post_side", lambda h: self.side.forward(h, batch)))
        for i, (role, sublayer) in enumerate(run):
            then = self.reader if i + 1 < len(run) else next_pre
            h = self.norms[role].add_normed(x, sublayer(h), then=then, out_dtype=dt)
        return h

    def first_norm(self):
        return self.reader


class ShiftedReader:
    """What a run of a :class:`NormedSumBlock` reads first: the stream in the compute dtype and, for the mixer, its rows
    shifted towards the row before (the same tensor where the block shifts nothing)."""
    graph_safe = True

    def __init__(self, block, view, batch):
        self.block, self.view, self.batch = block, view, batch

    def forward(self, x, out_dtype, rows=None):
        blk = self.block
        y = x if out_dtype == torch.float32 else torch.empty_like(x, dtype=out_dtype)
        if blk.shift is None:
            if y is not x:
                kernels.cast_rows(y, x)
            return y, y
        h = torch.empty_like(x, dtype=out_dtype)
        kernels.token_shift(h, x, blk.shift, self.view.block_state, self.batch, y=y if y is not x else None)
        return y, h

    def outputs(self, x, out_dtype):
        """(the arguments that make :func:`kernels.norm_of_sum` write what this reader reads, the tensors it writes),
        for a step of single tokens (or a block that shifts nothing)."""
        blk = self.block
        y = x if out_dtype == torch.float32 else torch.empty_like(x, dtype=out_dtype)
        args = {} if y is x else {"y": y}
        if blk.shift is None:
            return args, (y, y)
        h = torch.empty_like(x, dtype=out_dtype)
        args.update(shifted=h, shift=blk.shift, prev=self.view.block_state, slots=self.batch.slots)
        return args, (y, h)


@register_part("block", "normed_sum")
class NormedSumBlock(Block):
    """Parameters: ``hidden_size``, ``alpha``; optional ``shift_weight`` (tensor name, [hidden]) and ``gates``: for the
    mixer and for the feed-forward {``weight`` ([hidden, hidden]), ``bias`` ([hidden])} of tensor names, or None.
    Norm roles ``mixer_sum`` and ``feed_forward_sum`` (``layer_norm``).  A layer whose feed-forward is of the kind
    ``none`` has the first half only."""
    roles = ("mixer_sum", "feed_forward_sum")

    def __init__(self, params, ctx, mixer, feed_forward, norms):
        if not feed_forward.present:
            self.roles = ("mixer_sum",)
        super().__init__(params, ctx, mixer, feed_forward, norms)
        self.hidden = int(self.param("hidden_size"))
        self.alpha = float(self.param("alpha"))
        self.shift_name = self.params.get("shift_weight")
        halves = 2 if feed_forward.present else 1
        self.gate_names = [g for g in (self.params.get("gates") or [None, None])][:halves]
        for n in norms.values():
            if not isinstance(n, LayerNorm):
                raise ConfigError("normed_sum: the norms of the sums are of the kind layer_norm")
        self.shift = None
        self.gates = [None] * halves

    def state_need(self):
        return StateNeed((self.hidden,)) if self.shift_name else None

    def weight_decls(self):
        h, decls = self.hidden, super().weight_decls()
        if self.shift_name:
            decls.append(WeightDecl(self.shift_name, (h,), "blend"))
        for g in self.gate_names:
            if g is not None:
                decls += [WeightDecl(g["weight"], (h, h)), WeightDecl(g["bias"], (h,), "norm")]
        return decls

    def load(self, weights):
        super().load(weights)
        if self.shift_name:
            self.shift = weights[self.shift_name].to(torch.float32).contiguous()
        for q, g in enumerate(self.gate_names):
            if g is not None:
                self.gates[q] = (weights[g["weight"]].to(self.ctx.compute_dtype).contiguous(),
                                 weights[g["bias"]].to(torch.float32).contiguous())

    def _gate_numel(self) -> int:
        return sum(self.hidden * self.hidden for g in self.gate_names if g is not None)

    def decode_bytes(self, lens) -> int:
        state = len(lens) * 2 * 4 * self.hidden if self.shift_name else 0
        el = 4 if self.ctx.compute_dtype == torch.float32 else 2
        return super().decode_bytes(lens) + self._gate_numel() * el + state

    def prefill_flops(self, lens) -> int:
        return super().prefill_flops(lens) + 2 * sum(lens) * self._gate_numel()

    def first_norm(self):
        raise ConfigError("normed_sum: what a run reads first depends on its state (see Block.first_read)")

    def first_read(self, view, batch):
        return ShiftedReader(self, view, batch)

    def _gate(self, which: int, y):
        """The arguments that put this sublayer's gate into the kernel of its residual sum."""
        if self.gates[which] is None:
            return {}
        w, b = self.gates[which]
        z = linear_split(y, w, wide=True)
        return {"gate": z.parts if isinstance(z, PartialSums) else z, "gate_bias": b}

    def forward(self, x, batch, view, normed=None, next_pre=None):
        dt = self.ctx.compute_dtype
        y, h = normed if normed is not None else ShiftedReader(self, view, batch).forward(x, dt)
        gate = self._gate(0, y)
        a = self.mixer.forward(h, batch, view)
        if not self.feed_forward.present:
            return self._close(self.norms["mixer_sum"], x, a, gate, batch, next_pre)
        y = x if dt == torch.float32 else torch.empty_like(x, dtype=dt)
        self.norms["mixer_sum"].of_sum(x, a, self.alpha, y=None if y is x else y, **gate)
        gate = self._gate(1, y)
        return self._close(self.norms["feed_forward_sum"], x, self.feed_forward.forward(y, batch), gate, batch, next_pre)

    def _close(self, norm, x, a, gate, batch, next_pre):
        """The layer's last residual sum; returns what ``next_pre`` reads of the new stream."""
        dt = self.ctx.compute_dtype
        if isinstance(next_pre, ShiftedReader) and (not batch.is_prefill or next_pre.block.shift is None):
            args, out = next_pre.outputs(x, dt)
            norm.of_sum(x, a, self.alpha, **gate, **args)
            return out
        # a prompt: a row's shift wants its neighbour's new row, which another block of the kernel makes
        norm.of_sum(x, a, self.alpha, **gate)
        return None if next_pre is None else next_pre.forward(x, dt)

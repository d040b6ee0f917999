"""Arrangements of parts into a block.

"prenorm" (crates/model/src/llama.rs:264-271): x += mixer(norm1(x)); x += feed_forward(norm2(x)).
The residual stream is float32; each addition is fused into the norm that follows it, so a block
takes (resid, pending delta) and returns (resid, its own pending delta).

In steps of a few rows a norm is a kernel that moves a few kilobytes.  Where the parts on both
sides of a norm say that they can (`Part.fuses_norms`) and the norm offers it (`Norm.sink`), the
block hands the norm's sink to the part before it, which adds its result to the residual stream in
its last product, and passes the `ops.ScaledRows` it gets back to the part after it, whose first
product applies the scale; "pending" is then such rows instead of a delta.  The same holds across
blocks: the model names the next block, and `entry_sink` answers for its first norm."""

from __future__ import annotations

import torch

from .. import ops
from ..ops.profile import span
from .base import (Part, ProjectedMixer, build_feed_forward, build_mixer, build_norm, register_arrangement)


class PreNormBlock:
    def __init__(self, spec, dtype, device):
        self.norm1 = build_norm(spec.norm1, dtype, device)
        self.mixer = build_mixer(spec.mixer, dtype, device)
        # a layer may have no feed-forward: its mixer's result is then the block's pending addition
        self.feed_forward = build_feed_forward(spec.feed_forward, dtype, device) if spec.feed_forward is not None else None
        self.norm2 = build_norm(spec.norm2, dtype, device) if self.feed_forward is not None else None

    def parts(self):
        return tuple(p for p in (self.norm1, self.mixer, self.norm2, self.feed_forward) if p is not None)

    chains_norms = True      # `forward` takes `next_block`

    def entry_sink(self, resid, step):
        """For the block that runs before this one: the sink of this block's first norm, if its
        mixer takes the rows that come out of it."""
        return self.norm1.sink(resid, step) if self.mixer.fuses_norms(step) else None

    def forward(self, resid, pending, step, cache, state, writes_cache=True, next_block=None):
        h = pending if isinstance(pending, ops.ScaledRows) else self.norm1.forward(resid, pending, step)
        if self.feed_forward is None:
            sink = next_block.entry_sink(resid, step) if self.mixer.fuses_norms(step) and next_block is not None else None
            if sink is not None:
                return resid, self.mixer.forward(h, step, cache, state, writes_cache, sink=sink)
            return resid, self.mixer.forward(h, step, cache, state, writes_cache)
        mixer_fuses, ff_fuses = self.mixer.fuses_norms(step), self.feed_forward.fuses_norms(step)
        sink = self.norm2.sink(resid, step) if mixer_fuses and ff_fuses else None
        if sink is not None:
            h = self.mixer.forward(h, step, cache, state, writes_cache, sink=sink)
        else:
            a = self.mixer.forward(h, step, cache, state, writes_cache)
            h = self.norm2.forward(resid, a, step)
        sink = next_block.entry_sink(resid, step) if ff_fuses and next_block is not None else None
        if sink is not None:
            return resid, self.feed_forward.forward(h, step, sink=sink)
        return resid, self.feed_forward.forward(h, step)


class SandwichBlock:
    """x += scale1 * post_norm1(mixer(norm1(x))); x += scale2 * post_norm2(feed_forward(norm2(x))),
    the second line only when the layer has a feed-forward.  The residual stream and both norms of
    a sublayer's result are float32: one kernel norms the result, scales it, adds it to the stream
    and norms the stream for the sublayer that follows, also when that is the first sublayer of the
    next block of this kind (the block then returns those rows as `NormedRows`).  A block returns no
    pending delta: its additions are done when it returns."""

    def __init__(self, spec, dtype, device):
        self.dtype = dtype
        self.norm1 = build_norm(spec.norm1, dtype, device)
        self.mixer = build_mixer(spec.mixer, dtype, device)
        self.post_norm1 = build_norm(spec.post_norm1, dtype, device)
        self.scale1_name, self.scale2_name = spec.scale1, spec.scale2
        self.hidden = spec.norm1.dim
        self.feed_forward = build_feed_forward(spec.feed_forward, dtype, device) if spec.feed_forward is not None else None
        self.norm2 = build_norm(spec.norm2, dtype, device) if self.feed_forward is not None else None
        self.post_norm2 = build_norm(spec.post_norm2, dtype, device) if self.feed_forward is not None else None
        self.scale1 = self.scale2 = None
        for n in (self.norm1, self.post_norm1, self.norm2, self.post_norm2):
            if n is not None and not hasattr(n, "weight"):
                raise ValueError("the sandwich arrangement takes norms that are a weight and an eps (RMSNorm)")

    chains_norms = True      # `forward` takes `next_block`

    def entry_sink(self, resid, step):
        return None          # nothing is left to the product before this block

    def parts(self):
        own = _BlockTensors(self)
        return tuple(p for p in (self.norm1, self.mixer, self.post_norm1, self.norm2, self.feed_forward,
                                 self.post_norm2, own) if p is not None)

    def _last(self, sub, resid, post_norm, scale, step, next_block, bias=None):
        """The block's last addition; norms the stream for the next block when that is a sandwich too."""
        if isinstance(next_block, SandwichBlock):
            h = step.buffer("norm_out", (resid.shape[0], self.hidden), self.dtype)
            ops.post_norm_residual(sub, resid, post_norm.weight, post_norm.eps, scale, bias=bias,
                                   w_next=next_block.norm1.weight, eps_next=next_block.norm1.eps, out=h)
            return resid, NormedRows(h)
        ops.post_norm_residual(sub, resid, post_norm.weight, post_norm.eps, scale, bias=bias)
        return resid, None

    def forward(self, resid, pending, step, cache, state, writes_cache=True, next_block=None):
        h = pending.x if isinstance(pending, NormedRows) else self.norm1.forward(resid, pending, step)
        a = self.mixer.forward(h, step, cache, state, writes_cache)
        if self.feed_forward is None:
            return self._last(a, resid, self.post_norm1, self.scale1, step, next_block)
        h = step.buffer("norm_out", (resid.shape[0], self.hidden), self.dtype)
        ops.post_norm_residual(a, resid, self.post_norm1.weight, self.post_norm1.eps, self.scale1,
                               w_next=self.norm2.weight, eps_next=self.norm2.eps, out=h)
        defer = getattr(self.feed_forward, "b_down", None) is not None
        f = self.feed_forward.forward(h, step, defer_bias=True) if defer else self.feed_forward.forward(h, step)
        return self._last(f, resid, self.post_norm2, self.scale2, step, next_block,
                          bias=self.feed_forward.b_down if defer else None)


class OutNormBlock:
    """x += m * norm1(mixer(x)); x += m * norm2(feed_forward(x)), the second line only when the layer has a
    feed-forward.  The sublayers read the stream as it is, and only their results are normed.  The stream
    and the norms are float32: one kernel norms a result, adds it to the stream and leaves the stream,
    rounded to the compute type, for the sublayer that follows (in float32 that sublayer reads the stream
    itself).  A block returns no pending delta, and hands the next block of its kind the rounded stream."""

    def __init__(self, spec, dtype, device):
        self.dtype = dtype
        self.mult = float(spec.residual_mult)
        self.hidden = spec.norm1.dim
        self.mixer = build_mixer(spec.mixer, dtype, device)
        self.norm1 = build_norm(spec.norm1, dtype, device)
        self.feed_forward = build_feed_forward(spec.feed_forward, dtype, device) if spec.feed_forward is not None else None
        self.norm2 = build_norm(spec.norm2, dtype, device) if self.feed_forward is not None else None
        for n in (self.norm1, self.norm2):
            if n is not None and not hasattr(n, "weight"):
                raise ValueError("the outnorm arrangement takes norms that are a weight and an eps (RMSNorm)")

    chains_norms = True      # `forward` takes `next_block`

    def entry_sink(self, resid, step):
        return None

    def parts(self):
        return tuple(p for p in (self.mixer, self.norm1, self.feed_forward, self.norm2) if p is not None)

    def _stream(self, resid, step):
        """The stream as a sublayer reads it."""
        if self.dtype == torch.float32:
            return resid
        h = step.buffer("stream_copy", (resid.shape[0], self.hidden), self.dtype)
        return ops.post_norm_residual(None, resid, None, 0.0, out=h)

    def _join(self, sub, norm, resid, step, wanted: bool):
        """resid += m * norm(sub); returns the stream for the next sublayer if one is `wanted`."""
        if not wanted or self.dtype == torch.float32:
            ops.post_norm_residual(sub, resid, norm.weight, norm.eps, mult=self.mult)
            return resid if wanted else None
        h = step.buffer("stream_copy", (resid.shape[0], self.hidden), self.dtype)
        return ops.post_norm_residual(sub, resid, norm.weight, norm.eps, mult=self.mult, out=h)

    def forward(self, resid, pending, step, cache, state, writes_cache=True, next_block=None):
        h = pending.x if isinstance(pending, StreamRows) else self._stream(resid, step)
        a = self.mixer.forward(h, step, cache, state, writes_cache)
        chained = isinstance(next_block, OutNormBlock) and next_block.dtype == self.dtype
        if self.feed_forward is None:
            h = self._join(a, self.norm1, resid, step, chained)
        else:
            h = self._join(a, self.norm1, resid, step, True)
            f = self.feed_forward.forward(h, step)
            h = self._join(f, self.norm2, resid, step, chained)
        return resid, (StreamRows(h) if chained else None)


class PostNormBlock:
    """x = norm1(a x + mixer(x)); x = norm2(a x + feed_forward(x)), the second line only when the layer has a
    feed-forward; a is a constant.  The sublayers read the stream as it is.  The stream, the sums and the norms
    are float32: one kernel adds a sublayer's result to the scaled stream, norms the sum into the stream and
    leaves the stream, rounded to the compute type, for the sublayer that follows (in float32 that sublayer reads
    the stream itself).  A mixer of several branches (`forward_branches`) has its branches normed and averaged in
    the same kernel.  A block returns no pending delta, and hands the next block of its kind the rounded stream."""

    def __init__(self, spec, dtype, device):
        self.dtype = dtype
        self.alpha = float(spec.stream_mult)
        self.hidden = spec.norm1.dim
        self.mixer = build_mixer(spec.mixer, dtype, device)
        self.norm1 = build_norm(spec.norm1, dtype, device)
        self.feed_forward = build_feed_forward(spec.feed_forward, dtype, device) if spec.feed_forward is not None else None
        self.norm2 = build_norm(spec.norm2, dtype, device) if self.feed_forward is not None else None
        for n in (self.norm1, self.norm2):
            if n is not None and not hasattr(n, "weight"):
                raise ValueError("the postnorm arrangement takes norms that are a weight and an eps (RMSNorm)")

    chains_norms = True      # `forward` takes `next_block`

    def entry_sink(self, resid, step):
        return None

    def parts(self):
        return tuple(p for p in (self.mixer, self.norm1, self.feed_forward, self.norm2) if p is not None)

    def _stream(self, resid, step):
        if self.dtype == torch.float32:
            return resid
        h = step.buffer("stream_copy", (resid.shape[0], self.hidden), self.dtype)
        return ops.post_norm_residual(None, resid, None, 0.0, out=h)

    def _join(self, terms, eps_branch, norm, resid, step, wanted: bool):
        """resid = norm(alpha * resid + sum of the terms); returns the stream for the next sublayer if `wanted`."""
        h = None
        if wanted and self.dtype != torch.float32:
            h = step.buffer("stream_copy", (resid.shape[0], self.hidden), self.dtype)
        ops.sum_norm(resid, self.alpha, terms, norm.weight, norm.eps, out=h, eps_branch=eps_branch)
        return (h if h is not None else resid) if wanted else None

    def forward(self, resid, pending, step, cache, state, writes_cache=True, next_block=None):
        h = pending.x if isinstance(pending, StreamRows) else self._stream(resid, step)
        chained = isinstance(next_block, (PostNormBlock, OutNormBlock)) and next_block.dtype == self.dtype
        branches = getattr(self.mixer, "forward_branches", None)
        if branches is not None and len(self.mixer.branches) <= 2:      # the joining kernel takes two terms
            terms, eps_b = branches(h, step, cache, state, writes_cache)
        else:
            terms, eps_b = [(self.mixer.forward(h, step, cache, state, writes_cache), None, 1.0)], 0.0
        h = self._join(terms, eps_b, self.norm1, resid, step, chained or self.feed_forward is not None)
        if self.feed_forward is not None:
            f = self.feed_forward.forward(h, step)
            h = self._join([(f, None, 1.0)], 0.0, self.norm2, resid, step, chained)
        return resid, (StreamRows(h) if chained else None)


class ParallelBlock:
    """h = norm1(x); x += mixer(h) + feed_forward(h), the second term only when the layer has a feed-forward.  The residual
    stream and the sums are float32: the two results are the block's pending additions (a pair), which the next norm joins.

    In steps of a few rows a block with a `ProjectedMixer` and a gated unit is two products around the mixer and no norm: the
    mixer's first matrix and gate|up lie in one stacked matrix, whose product applies the norm and gates its second part; the
    mixer's and the unit's last products are one product with two sources, which adds to the stream and feeds the next norm."""

    chains_norms = True      # `forward` takes `next_block`

    def __init__(self, spec, dtype, device):
        self.norm1 = build_norm(spec.norm1, dtype, device)
        self.mixer = build_mixer(spec.mixer, dtype, device)
        self.feed_forward = build_feed_forward(spec.feed_forward, dtype, device) if spec.feed_forward is not None else None
        if spec.norm2 is not None:
            raise ValueError("sublayers side by side have one norm")
        self.joint = _JointInput(self) if isinstance(self.mixer, ProjectedMixer) and hasattr(self.feed_forward, "w_gate_up") else None

    def parts(self):
        return tuple(p for p in (self.norm1, self.mixer, self.feed_forward, self.joint) if p is not None)

    def _fuses(self, step) -> bool:
        if self.feed_forward is None:
            return self.mixer.fuses_norms(step)
        return self.joint is not None and self.joint.w is not None and self.mixer.fuses_norms(step) \
            and self.feed_forward.fuses_norms(step)

    def entry_sink(self, resid, step):
        return self.norm1.sink(resid, step) if self._fuses(step) else None

    def forward(self, resid, pending, step, cache, state, writes_cache=True, next_block=None):
        h = pending if isinstance(pending, ops.ScaledRows) else self.norm1.forward(resid, pending, step)
        fuses = self._fuses(step)
        sink = next_block.entry_sink(resid, step) if fuses and next_block is not None else None
        if self.feed_forward is None:
            if sink is not None:
                return resid, self.mixer.forward(h, step, cache, state, writes_cache, sink=sink)
            return resid, self.mixer.forward(h, step, cache, state, writes_cache)
        if not fuses:
            return resid, (self.mixer.forward(h, step, cache, state, writes_cache), self.feed_forward.forward(h, step))
        ff = self.feed_forward
        with span("mixer in proj, mlp gate+up"):
            proj, act = ops.stream_gemm(h, self.joint.w, n_plain=self.joint.n_plain, slope=ff.slope, cubic=ff.cubic)
        heads = self.mixer.mix(proj, step, cache, state, writes_cache)
        with span("o proj + mlp down proj"):
            if sink is not None:
                sink.exact = True            # the two results were never rounded apart
                return resid, ops.linear(heads, self.mixer.w_o, sink=sink, second=(act, ff.w_down))
            return resid, (ops.linear(heads, self.mixer.w_o), ops.linear(act, ff.w_down))


class _JointInput(Part):
    """The matrices that read a parallel block's normed input, one below the other: the mixer's, then gate|up.  The two
    parts keep views of it."""

    graph_safe = True

    def __init__(self, block):
        self.block = block
        self.w = None

    def load(self, src) -> None:
        mixer, ff = self.block.mixer, self.block.feed_forward
        if mixer.w_in.dtype != torch.bfloat16 or getattr(ff, "interleave", 0) != 4 or ff.b_gate_up is not None or ff.b_down is not None:
            return
        self.n_plain = mixer.w_in.shape[0]
        self.w = torch.cat([mixer.w_in, ff.w_gate_up], dim=0).contiguous()
        mixer.w_in, ff.w_gate_up = self.w[:self.n_plain], self.w[self.n_plain:]


class StreamJoin(Part):
    """x <- W [x | x0], x0 being the stream as the embedding left it (`step.carry`): what a pass over looped layers starts with.
    Run between two blocks like a block without a cache.  With W = [W_x | W_0], W_0 x0 is the same on every pass of a step and
    worked out once; a pass then costs W_x x.  The stream goes into the product rounded to the compute type, its new value is
    float32.  In steps of a few rows the block before leaves the rounded stream (a sink with a weight of ones), and the product
    adds W_0 x0 and feeds the first norm of the block after."""

    graph_safe = True
    chains_norms = True

    EMBEDDED = "stream.embedded"

    def __init__(self, spec, dtype, device):
        self.spec = spec
        self.dtype = dtype
        self.ones = torch.ones((spec.hidden,), dtype=torch.float32, device=device)
        self.base_key = "stream_join." + spec.weight

    def tensors(self) -> dict:
        return {self.spec.weight: (self.spec.hidden, 2 * self.spec.hidden)}

    def load(self, src) -> None:
        w, n = src.get(self.spec.weight), self.spec.hidden
        self.w_x, self.w_0 = w[:, :n].contiguous(), w[:, n:].contiguous()

    def parts(self):
        return (self,)

    def fuses_norms(self, step) -> bool:
        return ops.fuses_norms(step.n_tokens, self.dtype, self.spec.hidden)

    def entry_sink(self, resid, step):
        return ops.ResidualSink(resid, self.ones, 0.0) if self.fuses_norms(step) else None

    def _stream(self, resid, pending, step):
        """The complete stream in the compute type."""
        if isinstance(pending, ops.ScaledRows):
            return pending.x
        deltas = pending if isinstance(pending, tuple) else (pending,) if pending is not None else ()
        h = step.buffer("stream_copy", (resid.shape[0], self.spec.hidden), self.dtype) if self.dtype != torch.float32 else None
        if deltas or h is not None:
            ops.sum_norm(resid, 1.0, [(d, None, 1.0) for d in deltas], None, 0.0, out=h)
        return h if h is not None else resid

    def forward(self, resid, pending, step, cache=None, state=None, writes_cache=True, next_block=None):
        with span("stream + embedding"):
            x = self._stream(resid, pending, step)
            base = step.carry.get(self.base_key)
            if base is None:
                base = step.carry[self.base_key] = ops.linear(step.carry[self.EMBEDDED], self.w_0, out_dtype=torch.float32)
            sink = next_block.entry_sink(resid, step) if self.fuses_norms(step) and next_block is not None else None
            if isinstance(sink, ops.ResidualSink):
                sink.base, sink.exact = base, True
                return resid, ops.linear(x, self.w_x, sink=sink)
            return ops.linear_add(x, self.w_x, base), None


class HyperBlock:
    """Pre-norm sublayers over S residual streams (hyper-connections).  A sublayer reads norm(sum_s read[s] x_s); its
    result y goes back by x_t <- sum_s mix[s, t] x_s + write[t] y, old streams on the right.  The streams are float32: one
    kernel updates them with a sublayer's result and makes the normed input of the sublayer that follows, also when that
    is the first sublayer of the next block of this kind (a block returns `Streams` with that update pending).  The
    streams start equal, so the first kernel reads the embedding's row as every stream.  In steps of a few rows, where
    the norm that follows needs no statistics, the part's last product does the update and the norm in its epilogue
    (`ops.StreamsSink`).  After the last block the final norm reads the sum of the streams; a block of another
    arrangement that follows gets that sum as its residual stream."""

    chains_norms = True      # `forward` takes `next_block`

    def __init__(self, spec, dtype, device):
        self.dtype = dtype
        self.hidden = spec.norm1.dim
        self.norm1 = build_norm(spec.norm1, dtype, device)
        self.mixer = build_mixer(spec.mixer, dtype, device)
        self.feed_forward = build_feed_forward(spec.feed_forward, dtype, device) if spec.feed_forward is not None else None
        self.norm2 = build_norm(spec.norm2, dtype, device) if self.feed_forward is not None else None
        if spec.hyper1 is None or (self.feed_forward is not None and spec.hyper2 is None):
            raise ValueError("the hyper arrangement takes the coefficients of every sublayer (HyperSpec)")
        self.streams = int(spec.hyper1.streams)
        if not 1 <= self.streams <= ops.MAX_STREAMS:
            raise ValueError(f"one to {ops.MAX_STREAMS} residual streams, got {self.streams}")
        if self.feed_forward is not None and int(spec.hyper2.streams) != self.streams:
            raise ValueError("both sublayers of a block run over the same streams")
        self.hyper1 = _HyperTensors(spec.hyper1)
        self.hyper2 = _HyperTensors(spec.hyper2) if self.feed_forward is not None else None
        for n in (self.norm1, self.norm2):
            if n is not None and not hasattr(n, "stream_norm"):
                raise ValueError("the hyper arrangement takes norms that `ops.stream_mix` knows")

    def entry_sink(self, resid, step):
        return None          # nothing of an ordinary residual stream is left to the product before this block

    def entry_streams(self, step, n_streams: int):
        """For the part that runs before this block over the same streams: what it would have to read them with."""
        return (self.hyper1.read, self.norm1) if n_streams == self.streams else None

    def parts(self):
        return tuple(p for p in (self.hyper1, self.norm1, self.mixer, self.hyper2, self.norm2, self.feed_forward)
                     if p is not None)

    def _join(self, part, run, streams, hyper, step, follows, bias=None):
        """Runs a sublayer and hands its result to the streams: in its last product where that can, else pending."""
        if follows is not None and part.fuses_norms(step):
            sink = streams.sink(hyper, follows, step, self.dtype)
            if sink is not None:
                return streams.normed_by(run(sink=sink), sink)
        return streams.pending(run() if bias is None else run(defer_bias=True), bias, hyper)

    def forward(self, resid, pending, step, cache, state, writes_cache=True, next_block=None):
        if isinstance(pending, Streams):
            streams = pending
        else:
            if pending is not None:      # a block of another arrangement has left its last addition
                for delta in pending if isinstance(pending, tuple) else (pending,):
                    ops.stream_mix(resid, 1, y=delta, x_out=resid.unsqueeze(1))
            streams = Streams(resid, self.streams)
        ask = getattr(next_block, "entry_streams", None)
        after = ask(step, self.streams) if ask is not None else None
        h = streams.read((self.hyper1.read, self.norm1), step, self.dtype)
        mid = (self.hyper2.read, self.norm2) if self.feed_forward is not None else after
        streams = self._join(self.mixer, lambda **k: self.mixer.forward(h, step, cache, state, writes_cache, **k), streams,
                             self.hyper1, step, mid)
        if self.feed_forward is not None:
            h2 = streams.read(mid, step, self.dtype)
            streams = self._join(self.feed_forward, lambda **k: self.feed_forward.forward(h2, step, **k), streams,
                                 self.hyper2, step, after, getattr(self.feed_forward, "b_down", None))
        if ask is None:                  # whoever comes next knows nothing of streams
            streams.total(out=resid)
            return resid, None
        return resid, streams


class Streams:
    """The residual streams of a step between two sublayers: `x` float32 [T, S, W] (or [T, W]: one row that is every
    stream), perhaps with a sublayer's result still to be joined, or with the next sublayer's normed input already made."""

    def __init__(self, x, n: int, y=None, bias=None, hyper=None, rows=None):
        self.x, self.n, self.y, self.bias, self.hyper, self.rows = x, n, y, bias, hyper, rows

    def _update(self) -> dict:
        if self.y is None:
            return {}
        return {"y": self.y, "y_bias": self.bias, "mix": self.hyper.mix, "out_coef": self.hyper.write}

    def _home(self, step):
        return step.buffer("streams", (self.x.shape[0], self.n, self.x.shape[-1]), torch.float32)

    def pending(self, y, bias, hyper) -> "Streams":
        return Streams(self.x, self.n, y, bias, hyper)

    def normed_by(self, rows, sink) -> "Streams":
        return Streams(sink.x_out, self.n, rows=rows)

    def read(self, how, step, dtype):
        """The normed input of the sublayer that reads the streams by `how` = (coefficients, norm)."""
        if self.rows is not None:
            return self.rows
        coef, norm = how
        h = step.buffer("norm_out", (self.x.shape[0], self.x.shape[-1]), dtype)
        update = self._update()
        x_out = self._home(step) if update else None
        with span("streams + norm"):
            ops.stream_mix(self.x, self.n, x_out=x_out, in_coef=coef, norm=norm.stream_norm(), h=h, **update)
        if update:
            self.x, self.y = x_out, None
        return h

    def sink(self, hyper, follows, step, dtype):
        coef, norm = follows
        sn = norm.stream_norm()
        if sn.kind != "dynamic_tanh" or self.y is not None or not ops.fuses_norms(self.x.shape[0], dtype, self.x.shape[-1]):
            return None
        return ops.StreamsSink(self.x, self._home(step), self.n, hyper.mix, hyper.write, coef, sn)

    def normed_rows(self, norm, step, rows, dtype):
        """The rows `rows` of the streams' sum after `norm` (what the LM head reads)."""
        if self.rows is not None:        # made by the last product, for all rows of the step in order
            return self.rows
        out = step.buffer("norm_rows_out", (rows.shape[0], self.x.shape[-1]), dtype)
        with span("streams + norm"):
            return ops.stream_mix(self.x, self.n, norm=norm.stream_norm(), h=out, rows=rows, **self._update())

    def total(self, out=None):
        """The sum of the streams, float32 [T, W]."""
        out = out if out is not None else torch.empty((self.x.shape[0], self.x.shape[-1]), dtype=torch.float32, device=self.x.device)
        return ops.stream_mix(self.x, self.n, u_out=out, **self._update())


class _HyperTensors(Part):
    """The coefficients of one sublayer's hyper-connection."""

    graph_safe = True

    def __init__(self, spec):
        self.spec = spec

    def tensors(self) -> dict:
        s = self.spec
        return {s.read: (s.streams,), s.write: (s.streams,), s.mix: (s.streams, s.streams)}

    def load(self, src) -> None:
        s = self.spec
        self.read, self.write, self.mix = (src.get(n, "vector").contiguous() for n in (s.read, s.write, s.mix))


class StreamRows:
    """What an outnorm block hands the next one: `x`, the (complete) residual stream in the compute type."""

    def __init__(self, x):
        self.x = x


class NormedRows:
    """What a block hands the next one when it has already normed the stream for it: `x`, the next
    block's first norm applied to the (complete) residual stream."""

    def __init__(self, x):
        self.x = x


class _BlockTensors(Part):
    """The block's own tensors (the per-channel scales), loaded with its parts."""

    graph_safe = True

    def __init__(self, block):
        self.block = block

    def tensors(self) -> dict:
        b = self.block
        return {n: (b.hidden,) for n in (b.scale1_name, b.scale2_name if b.feed_forward is not None else None)
                if n is not None}

    def load(self, src) -> None:
        b = self.block
        b.scale1 = src.get(b.scale1_name, "vector") if b.scale1_name is not None else None
        b.scale2 = src.get(b.scale2_name, "vector") if (b.scale2_name is not None and b.feed_forward is not None) else None


register_arrangement("prenorm", PreNormBlock)
register_arrangement("sandwich", SandwichBlock)
register_arrangement("outnorm", OutNormBlock)
register_arrangement("postnorm", PostNormBlock)
register_arrangement("hyper", HyperBlock)
register_arrangement("parallel", ParallelBlock)
register_arrangement("stream_join", StreamJoin)

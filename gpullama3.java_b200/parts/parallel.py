"""Parts that stand side by side instead of one behind the other.

``ParallelBlock``: the mixer and the feed-forward read the same residual stream, each through a norm of its own, and both
results join it at once,

    x <- x + mixer(norm_1(x)) + feed_forward(norm_2(x))         (a layer may have no feed-forward, or one norm for both)

``ParallelMixers``: two mixers on the same input, each with a factor,  left_scale * left(h) + right_scale * right(h).

Parts whose result is one last product over rows they make (``OpenEnded``) are multiplied together: the mixers and the
feed-forward write their rows into neighbouring columns of one buffer and ONE product over the joined weights adds the
layer's whole result into the stream; two mixers likewise start with one product over their joined input weights, and so do a
mixer and a feed-forward that read the same norm and both give their first product away.  What a feed-forward adds to the stream
itself (a mixture's routed experts) it adds before that last product.  The
factors of ``ParallelMixers`` are applied to the rows in 32 bits.  The two norms differ in their weights alone, so a prompt
makes both in one read of the stream, and in a decode step the product that completes the stream leaves both copies for
the next block's products (``ScaledRows``), whose shared row factor they apply themselves.  In a decode step the
feed-forward's first product, which streams most of a layer's weights, runs on a stream of its own beside the mixer's short
kernels (a recorded step has two branches there, which meet in the layer's last product)."""
from __future__ import annotations

import torch

from ..config.base import ConfigError
from ..cache.sequence_cache import EntryNeeds
from ..kernels import ops
from .base import Block, Mixer, OpenEnded, StepContext, all_parts, register_block, register_mixer
from .linear import Linear


class NormPair:
    """Two norms of the same rows with one eps, as ``then_norm`` of the block before: its last product leaves the rows
    under both weights."""

    def __init__(self, first, second):
        self.first, self.second = first, second

    def row_factor_form(self):
        return self.first.row_factor_form()

    def second_form(self):
        return self.second.row_factor_form()[0]


def _as_pair(first, second) -> NormPair | None:
    """The two norms as a pair, if they differ in their weights alone."""
    a, b = first.row_factor_form(), second.row_factor_form()
    if a is None or b is None or a[1:] != b[1:] or a[0].dtype != b[0].dtype:
        return None
    return NormPair(first, second)


def _joined(outputs, device=None) -> Linear:
    """One product for several last products: weights side by side, biases added up."""
    weights = [w for w, _ in outputs]
    common = torch.float32 if any(w.dtype == torch.float32 for w in weights) else weights[0].dtype
    biases = [b for _, b in outputs if b is not None]
    bias = None
    if biases:
        bias = biases[0].clone()
        for b in biases[1:]:
            bias += b
    return Linear(torch.cat([w.to(common) for w in weights], dim=1).contiguous(), bias)


_side_streams: dict = {}


def _beside(device):
    """Launches inside run on a stream of their own behind everything the current stream holds so far, beside what it is
    given next, until ``_join``."""
    side = _side_streams.get(device)
    if side is None:
        side = _side_streams[device] = torch.cuda.Stream(device)
    side.wait_stream(torch.cuda.current_stream(device))
    return torch.cuda.stream(side)


def _join(device) -> None:
    """The current stream waits for what runs beside it."""
    torch.cuda.current_stream(device).wait_stream(_side_streams[device])


class ParallelBlock(Block):
    def __init__(self, mixer, mixer_norm, feed_forward=None, feed_forward_norm=None):
        """``feed_forward_norm`` None: mixer and feed-forward both read the rows of ``mixer_norm``."""
        if feed_forward is None and feed_forward_norm is not None:
            raise ConfigError("a norm of the feed-forward's input needs a feed-forward")
        given = {"mixer": mixer, "mixer_norm": mixer_norm, "feed_forward": feed_forward, "feed_forward_norm": feed_forward_norm}
        super().__init__(**{k: v for k, v in given.items() if v is not None})
        for k, v in given.items():
            setattr(self, k, v)
        self.out: Linear | None = None     # the joined last product, where every part gives its own away
        self.inputs: Linear | None = None  # the joined first product, where both parts read one norm and give theirs away

    def after_load(self):
        sublayers = [p for p in (self.mixer, self.feed_forward) if p is not None]
        if all(isinstance(p, OpenEnded) for p in sublayers):
            self.columns = [p.open_columns() for p in sublayers]
            self.out = _joined([p.take_output() for p, n in zip(sublayers, self.columns) if n])
            if self.shares_norm and all(p.gives_input for p in sublayers):
                ins = [p.take_input() for p in sublayers]
                common = torch.float32 if any(w.dtype == torch.float32 for w in ins) else ins[0].dtype
                self.input_columns = ins[0].shape[0]
                self.inputs = Linear(torch.cat([w.to(common) for w in ins], dim=0).contiguous())

    @property
    def shares_norm(self) -> bool:
        return self.feed_forward is not None and self.feed_forward_norm is None

    @property
    def graph_safe(self):
        return all(p.graph_safe for p in all_parts(self).values())

    @property
    def pad_safe(self):
        return all(p.pad_safe for p in all_parts(self).values())

    def first_norm(self):
        if self.feed_forward_norm is None:
            return self.mixer_norm
        return _as_pair(self.mixer_norm, self.feed_forward_norm)

    def takes_scaled_rows(self, ctx: StepContext) -> bool:
        first = self.first_norm()
        return (self.out is not None and first is not None and first.row_factor_form() is not None
                and all(p.takes_scaled_rows(ctx) for p in (self.mixer, self.feed_forward) if p is not None))

    def leaves_scaled_rows(self, ctx: StepContext) -> bool:
        return ctx.all_decode and self.out is not None

    def _normed(self, residual, ctx: StepContext):
        """The inputs of the mixer and the feed-forward (None without one)."""
        if self.feed_forward_norm is None:
            h = self.mixer_norm.forward(residual, ctx.dtype, alloc=ctx.empty)
            return h, h
        pair = _as_pair(self.mixer_norm, self.feed_forward_norm)
        if pair is not None and pair.second_form().dtype == torch.float32:
            weight, eps, _ = pair.row_factor_form()
            outs = [ctx.empty(residual.shape, ctx.dtype) for _ in range(2)]
            ops.rmsnorm_pair(residual, (weight, pair.second_form()), outs, eps)
            return outs
        return (self.mixer_norm.forward(residual, ctx.dtype, alloc=ctx.empty),
                self.feed_forward_norm.forward(residual, ctx.dtype, alloc=ctx.empty))

    def forward(self, residual, ctx: StepContext, cache, writes_cache=True, x_in=None, then_norm=None):
        if x_in is None:
            h, g = self._normed(residual, ctx)
        else:
            h, g = x_in if isinstance(x_in, tuple) else (x_in, x_in)
        if self.out is None:    # (a part that keeps its last product to itself: one after the other, both inputs made before)
            self.mixer.forward(h, ctx, cache, residual, writes_cache)
            if self.feed_forward is not None:
                self.feed_forward.forward(g, ctx, residual)
            return None
        rows = ctx.empty((residual.shape[0], self.out.in_features), ctx.dtype)
        n = self.columns[0]
        if self.feed_forward is None:
            self.mixer.rows_into(h, ctx, cache, rows, writes_cache)
            return self.out.add_to(rows, residual, then_norm)
        raw = self.inputs.store(h, ctx.dtype, ctx.empty) if self.inputs is not None else None

        def mix():
            if raw is not None:
                self.mixer.rows_from(raw[:, :self.input_columns], ctx, cache, rows[:, :n], writes_cache)
            else:
                self.mixer.rows_into(h, ctx, cache, rows[:, :n], writes_cache)

        def feed_forward():
            if raw is not None:
                self.feed_forward.rows_from(raw[:, self.input_columns:], ctx, None, rows[:, n:])
            elif self.columns[1]:
                self.feed_forward.rows_into(g, ctx, None, rows[:, n:])
            self.feed_forward.adds_itself(g, ctx, residual)

        if ctx.all_decode:
            with _beside(ctx.device):
                feed_forward()
            mix()
            _join(ctx.device)
        else:
            mix()
            feed_forward()
        return self.out.add_to(rows, residual, then_norm)


class ParallelMixers(Mixer, OpenEnded):
    def __init__(self, left, right, left_scale: float = 1.0, right_scale: float = 1.0):
        for name, m in (("left", left), ("right", right)):
            if not (isinstance(m, OpenEnded) and isinstance(m, Mixer)):
                raise ConfigError(f"parallel mixers: the {name} mixer keeps its products to itself")
        self.left, self.right = left, right
        self.scales = (float(left_scale), float(right_scale))
        self.inputs: Linear | None = None
        self.o: Linear | None = None

    @property
    def _both(self):
        return (("left", self.left), ("right", self.right))

    def children(self):
        return dict(self._both)

    @property
    def graph_safe(self):
        return self.left.graph_safe and self.right.graph_safe

    @property
    def pad_safe(self):
        return self.left.pad_safe and self.right.pad_safe

    def cache_need(self):
        needs = [(n, m.cache_need()) for n, m in self._both]
        needs = tuple((n, need) for n, need in needs if need is not None)
        return EntryNeeds(needs) if needs else None

    def after_load(self):
        ins = [m.take_input() for _, m in self._both]
        common = torch.float32 if any(w.dtype == torch.float32 for w in ins) else ins[0].dtype
        self.input_columns = [w.shape[0] for w in ins]
        self.inputs = Linear(torch.cat([w.to(common) for w in ins], dim=0).contiguous())
        self.columns = [m.open_columns() for _, m in self._both]
        self.o = _joined([m.take_output() for _, m in self._both])

    def open_columns(self):
        return sum(m.open_columns() for _, m in self._both)

    def take_output(self):
        weight, bias, self.o = self.o.weight, self.o.bias, None
        return weight, bias

    def take_input(self):
        weight, self.inputs = self.inputs.weight, None
        return weight

    def takes_scaled_rows(self, ctx: StepContext) -> bool:
        return ctx.all_decode and self.inputs is not None and self.inputs.links_with(ctx.n_tokens, ctx.dtype)

    def rows_into(self, x, ctx: StepContext, cache, rows, writes_cache=True, mul=1.0):
        self.rows_from(self.inputs.store(x, ctx.dtype, ctx.empty), ctx, cache, rows, writes_cache, mul)

    def rows_from(self, raw, ctx: StepContext, cache, rows, writes_cache=True, mul=1.0):
        at, col = 0, 0
        for (name, m), scale, n_in, n in zip(self._both, self.scales, self.input_columns, self.columns):
            view = cache.get(name) if isinstance(cache, dict) else None
            m.rows_from(raw[:, at:at + n_in], ctx, view, rows[:, col:col + n], writes_cache, scale * mul)
            at, col = at + n_in, col + n

    def forward(self, x, ctx: StepContext, cache, residual, writes_cache=True, then_norm=None):
        rows = ctx.empty((x.shape[0], self.open_columns()), ctx.dtype)
        self.rows_into(x, ctx, cache, rows, writes_cache)
        return self.o.add_to(rows, residual, then_norm)


register_block("parallel", ParallelBlock)
register_mixer("parallel", ParallelMixers)

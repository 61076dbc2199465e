"""Arrangements of a layer's parts around the residual stream.

`pre_norm` (student_engine.py:696-731):  h += mixer(norm_1(h));  h += feed_forward(norm_2(h)).
The stream `hidden` is float32 and is updated in place; a part's output (`delta`) is added to it by
the *next* norm's kernel, so a block takes the pending delta of the layer before it and returns its own."""
from __future__ import annotations

import torch

from .. import ops
from ..cache import BundleNeed
from .base import Norm, Part, Pending, PendingNormed, PendingPair, PendingScaled, PendingStreams, RowSum, fork, join, runs_side_by_side
from .registry import build_part, register_part


class PreNormBlock(Part):
    """Reads the layer spec's parts `mixer_norm`, `mixer` and, if the layer has a feed-forward, `feed_forward_norm` and
    `feed_forward`. With the layer spec's parameter `residual_mult` = m every sublayer's output enters the stream times m:
    h += m * mixer(norm_1(h));  h += m * feed_forward(norm_2(h))  (the product and the sum in float32, inside the next norm's
    kernel). A mixer may hand back two outputs under a factor each (`PendingScaled`); they go the same way."""

    accepts_pending = (PendingScaled,)

    def __init__(self, layer_spec):
        self.kind = "pre_norm"
        self.mixer_norm = build_part("norm", layer_spec.part("mixer_norm"))
        self.mixer = build_part("mixer", layer_spec.part("mixer"))
        self.feed_forward = self.feed_forward_norm = None
        if "feed_forward" in layer_spec.parts:
            self.feed_forward_norm = build_part("norm", layer_spec.part("feed_forward_norm"))
            self.feed_forward = build_part("feed_forward", layer_spec.part("feed_forward"))
        self.residual_mult = float(layer_spec.params.get("residual_mult", 1.0))

    def sub_parts(self):
        return [p for p in (self.mixer_norm, self.mixer, self.feed_forward_norm, self.feed_forward) if p is not None]

    def cache_need(self):
        return self.mixer.cache_need()

    def _forward_scaled(self, hidden, delta, ctx, site, writes_cache):
        """The layer with a residual multiplier, a mixer of two outputs, or no feed-forward: every output stays pending
        with its factor and is added, in float32, by the kernel of the norm that reads the stream next."""
        x = self.mixer_norm.forward(hidden, delta)
        delta = PendingScaled.of(self.mixer.forward(x, ctx, site, writes_cache), self.residual_mult)
        if self.feed_forward is None:
            return delta
        x = self.feed_forward_norm.forward(hidden, delta)
        return PendingScaled.of(self.feed_forward.forward(x, ctx), self.residual_mult)

    def forward(self, hidden, delta, ctx, site, writes_cache):
        if self.residual_mult != 1.0 or self.feed_forward is None or getattr(self.mixer, "scaled_outputs", False) \
                or isinstance(delta, PendingScaled):
            return self._forward_scaled(hidden, delta, ctx, site, writes_cache)
        rms = self.mixer_norm.fused_rms()
        if rms is not None and self.mixer.fused_takes(ctx):
            self.mixer.fused_forward(hidden, rms, ctx, site, writes_cache, delta)
            delta = None
        else:
            x = self.mixer_norm.forward(hidden, delta)
            delta = self.mixer.forward(x, ctx, site, writes_cache)
        rms = self.feed_forward_norm.fused_rms()
        if rms is not None and self.feed_forward.fused_takes(ctx):
            self.feed_forward.fused_forward(hidden, rms, ctx, delta)
            return None
        x = self.feed_forward_norm.forward(hidden, delta)
        return self.feed_forward.forward(x, ctx)


class SandwichBlock(Part):
    """Norms before AND after each sublayer:  h += post_1(mixer(norm_1(h)));  h += post_2(feed_forward(norm_2(h))).
    Reads the layer spec's parts `mixer_norm`, `mixer`, `mixer_post_norm` and, if the layer has a feed-forward,
    `feed_forward_norm`, `feed_forward`, `feed_forward_post_norm`. The norms after the sublayers must be plain RMS norms
    (`fused_rms`): each rides, with its addition into the stream, on the kernel of the norm that follows it
    (`ops.sandwich_norm`), the last one of a layer on the first norm of the next layer."""

    accepts_pending_normed = True

    def __init__(self, layer_spec):
        self.kind = "sandwich_norm"
        self.mixer_norm = build_part("norm", layer_spec.part("mixer_norm"))
        self.mixer = build_part("mixer", layer_spec.part("mixer"))
        self.mixer_post_norm = build_part("norm", layer_spec.part("mixer_post_norm"))
        self.feed_forward = self.feed_forward_norm = self.feed_forward_post_norm = None
        if "feed_forward" in layer_spec.parts:
            self.feed_forward_norm = build_part("norm", layer_spec.part("feed_forward_norm"))
            self.feed_forward = build_part("feed_forward", layer_spec.part("feed_forward"))
            self.feed_forward_post_norm = build_part("norm", layer_spec.part("feed_forward_post_norm"))
        for norm in (self.mixer_norm, self.mixer_post_norm, self.feed_forward_norm, self.feed_forward_post_norm):
            if norm is not None and type(norm).fused_rms is Norm.fused_rms:
                raise ValueError("sandwich_norm: the norms must be plain RMS norms")

    def sub_parts(self):
        return [p for p in (self.mixer_norm, self.mixer, self.mixer_post_norm, self.feed_forward_norm, self.feed_forward,
                            self.feed_forward_post_norm) if p is not None]

    def cache_need(self):
        return self.mixer.cache_need()

    def forward(self, hidden, delta, ctx, site, writes_cache):
        weight, eps = self.mixer_norm.fused_rms()
        if isinstance(delta, PendingNormed):
            x = torch.empty(hidden.shape, dtype=weight.dtype, device=hidden.device)
            delta.into(hidden, weight, eps, x)
        else:
            x = self.mixer_norm.forward(hidden, delta)
        y = self.mixer.forward(x, ctx, site, writes_cache)
        post = PendingNormed(y, *self.mixer_post_norm.fused_rms())
        if self.feed_forward is None:
            return post
        weight, eps = self.feed_forward_norm.fused_rms()
        x = torch.empty(hidden.shape, dtype=weight.dtype, device=hidden.device)
        post.into(hidden, weight, eps, x)
        # a feed-forward that leaves several rows per token hands them over unsummed: the next norm kernel adds them up
        run = getattr(self.feed_forward, "forward_rows", None) or self.feed_forward.forward
        return PendingNormed(run(x, ctx), *self.feed_forward_post_norm.fused_rms())


class ParallelBlock(Part):
    """Two sublayers side by side:  h = norm(x);  x += mixer(in(h)) + feed_forward(h);  or, with a norm for each,
    x += mixer(in(norm(x))) + feed_forward(feed_forward_norm(x)), both norms of the same x.
    Reads the layer spec's parts `norm`, `mixer` and, if the layer has them, `feed_forward`, `feed_forward_norm` and `mixer_input` (a
    part of role "mixer_input" that filters what the mixer reads and may keep a state of its own per sequence, such as a token
    shift; the feed-forward reads its norm's output as it is). The two outputs stay pending as a pair: the next norm kernel of a block
    of this kind adds their sum to the float32 stream on its way. In a block with two norms (plain RMS norms) that kernel makes both,
    and sums a feed-forward's unsummed rows as well; the two sublayers of a step of few rows then run on two streams."""

    accepts_pending = (PendingPair,)

    def __init__(self, layer_spec):
        self.kind = "parallel"
        self.norm = build_part("norm", layer_spec.part("norm"))
        self.mixer = build_part("mixer", layer_spec.part("mixer"))
        self.mixer_input = build_part("mixer_input", layer_spec.part("mixer_input")) if "mixer_input" in layer_spec.parts else None
        self.feed_forward = build_part("feed_forward", layer_spec.part("feed_forward")) if "feed_forward" in layer_spec.parts else None
        self.feed_forward_norm = build_part("norm", layer_spec.part("feed_forward_norm")) if "feed_forward_norm" in layer_spec.parts else None
        self.pair_norm = bool(getattr(self.norm, "takes_pair", False))   # its kernel adds two pending outputs on its way
        # plain RMS norms: one kernel for what is pending and up to two norms
        self.rms_norms = all(n is None or type(n).fused_rms is not Norm.fused_rms for n in (self.norm, self.feed_forward_norm))
        if self.feed_forward_norm is not None and (self.feed_forward is None or self.mixer_input is not None or not self.rms_norms):
            raise ValueError("parallel: a second norm goes with a feed-forward, with plain RMS norms and without a filter in front of the mixer")

    def sub_parts(self):
        return [p for p in (self.norm, self.mixer_input, self.mixer, self.feed_forward_norm, self.feed_forward) if p is not None]

    def cache_need(self):
        need = self.mixer.cache_need()
        if self.mixer_input is None or self.mixer_input.cache_need() is None:
            return need
        return BundleNeed((("input", self.mixer_input.cache_need()), ("mixer", need)))

    def _forward_rms(self, hidden, delta, ctx, site, writes_cache):
        """The layer with plain RMS norms (one or two) and nothing in front of the mixer."""
        weight, eps = self.norm.fused_rms()
        h1 = torch.empty(hidden.shape, dtype=weight.dtype, device=hidden.device)
        second = {}
        if self.feed_forward_norm is not None:
            weight2, eps2 = self.feed_forward_norm.fused_rms()
            second = {"weight2": weight2, "eps2": eps2, "out2": torch.empty_like(h1)}
        if isinstance(delta, PendingPair):
            ops.pair_rms_norm(hidden, delta.a, delta.b, weight, eps, h1, b_rows=delta.rows, **second)
        else:
            ops.pair_rms_norm(hidden, delta, None, weight, eps, h1, **second)
        if self.feed_forward is None:
            return PendingPair(self.mixer.forward(h1, ctx, site, writes_cache))
        h2 = second.get("out2", h1)
        # a feed-forward that leaves several rows per token hands them over unsummed: the next norm kernel adds them up
        run = getattr(self.feed_forward, "forward_rows", None) or self.feed_forward.forward
        if runs_side_by_side(h1):
            main, side = fork(h2)
            with torch.cuda.stream(side):
                fed = run(h2, ctx)
            mixed = self.mixer.forward(h1, ctx, site, writes_cache)
            join(main, side, *((fed.rows, fed.dest, fed.row_weight) if isinstance(fed, RowSum) else (fed,)))
        else:
            mixed, fed = self.mixer.forward(h1, ctx, site, writes_cache), run(h2, ctx)
        return PendingPair(mixed, fed)

    def forward(self, hidden, delta, ctx, site, writes_cache):
        if self.rms_norms and self.mixer_input is None:
            return self._forward_rms(hidden, delta, ctx, site, writes_cache)
        bundled = self.mixer_input is not None and self.mixer_input.cache_need() is not None
        if bundled and not writes_cache:
            raise ValueError("parallel: a layer whose mixer input keeps a state cannot read another entry's cache")
        # a mixer input that the norm's kernel can make on its way (single tokens): one launch for both
        rider = None
        if bundled and getattr(self.norm, "takes_shift", False) and hasattr(self.mixer_input, "rides_on_norm"):
            rider = self.mixer_input.rides_on_norm(hidden.shape[0], ctx, site["input"])
        extra = {} if rider is None else {"shift": rider}
        if isinstance(delta, PendingPair):
            if self.pair_norm and delta.rows is None:
                h = self.norm.forward(hidden, delta.a, delta.b, **extra)
            else:
                delta.add_to(hidden)
                h = self.norm.forward(hidden, None, **extra)
        else:
            h = self.norm.forward(hidden, delta, **extra)
        mixer_site, u = site, h
        if rider is not None:
            h, u = h
            mixer_site = site["mixer"]
        elif self.mixer_input is not None:
            u = self.mixer_input.forward(h, ctx, site["input"] if bundled else None)
            mixer_site = site["mixer"] if bundled else site
        mixed = self.mixer.forward(u, ctx, mixer_site, writes_cache)
        return PendingPair(mixed, self.feed_forward.forward(h, ctx) if self.feed_forward is not None else None)


class StreamsBlock(Part):
    """Several residual streams (hyper-connections): with X[0..n-1] the streams, all equal to the embedding's output at the start,
        u = sum_s a[s] X[s];   y = sublayer(filter(norm(u)));   X[r] <- sum_s M[s, r] X[s] + b[r] y
    for the mixer and then, if the layer has one, for the feed-forward, each with coefficients of its own. Reads the layer spec's
    parts `mixer_streams`, `mixer_norm`, `mixer` (and `mixer_input`, the filter, if there is one), and `feed_forward_streams`,
    `feed_forward_norm`, `feed_forward` (and `feed_forward_input`). What a sublayer leaves stays pending with its coefficients
    (`PendingStreams`): entering the streams, the next read, its norm and its filter are one kernel. The streams live between
    the blocks in the pending object; the model's `hidden` is the row they start from and receives their sum at the end."""

    accepts_pending = (PendingStreams,)

    def __init__(self, layer_spec):
        self.kind = "streams"
        part = lambda role, name: build_part(role, layer_spec.part(name)) if name in layer_spec.parts else None
        self.sublayers = []
        for name, role in (("mixer", "mixer"), ("feed_forward", "feed_forward")):
            if name in layer_spec.parts:
                self.sublayers.append((name, build_part("streams", layer_spec.part(name + "_streams")),
                                       build_part("norm", layer_spec.part(name + "_norm")), part("mixer_input", name + "_input"),
                                       build_part(role, layer_spec.part(name))))
        self.n = self.sublayers[0][1].streams
        if self.sublayers[0][0] != "mixer" or any(s[1].streams != self.n for s in self.sublayers):
            raise ValueError("streams: a layer has a mixer, and its sublayers work on as many streams")

    def sub_parts(self):
        return [p for _, *parts in self.sublayers for p in parts if p is not None]

    def cache_need(self):
        items = []
        for name, _, _, filter_, sublayer in self.sublayers:
            if filter_ is not None and filter_.cache_need() is not None:
                items.append((name + "_input", filter_.cache_need()))
            if name == "mixer" and sublayer.cache_need() is not None:
                items.append(("mixer", sublayer.cache_need()))
        return BundleNeed(tuple(items)) if items else None

    def forward(self, hidden, delta, ctx, site, writes_cache):
        if not writes_cache:
            raise ValueError("streams: a layer whose inputs keep a state cannot read another entry's cache")
        if not isinstance(delta, PendingStreams):
            if isinstance(delta, Pending):
                delta.add_to(hidden)
            elif delta is not None:
                ops.residual_add(hidden, delta)
            delta = PendingStreams(hidden, self.n)
        at = lambda name: site.get(name) if site is not None else None
        for name, streams, norm, filter_, sublayer in self.sublayers:
            x, source = delta.enter(streams, norm, filter_, ctx, at(name + "_input"))
            if name == "mixer":
                y = sublayer.forward(x, ctx, at("mixer"), True)
            else:   # a feed-forward that leaves several rows per token hands them over unsummed
                y = (getattr(sublayer, "forward_rows", None) or sublayer.forward)(x, ctx)
            delta = PendingStreams(source, self.n, y, streams)
        return delta


register_part("block", "streams", StreamsBlock)
register_part("block", "pre_norm", PreNormBlock)
register_part("block", "parallel", ParallelBlock)
register_part("block", "sandwich_norm", SandwichBlock)

"""Arrangements of parts in a layer.  ``PreNormBlock``:
``h = x + mixer(norm_1(x)); out = h + feed_forward(norm_2(h))``
(mlx_lm/models/gpt2.py:104-108).  The residual stream is updated in place by
the epilogues of the mixer's and the feed-forward's last products."""

from __future__ import annotations

import os
from typing import Optional

import torch

from .. import ops
from .base import VECTOR, Block, FeedForward, Init, Mixer, Norm, ParamSpec, Summands, register_part

# In bfloat16 a block lets its mixer and its feed-forward fold the norm before them into their first linear
# layer (parts/linear.py, ``Linear.fold_norm``): steps of few rows then run no norm kernels inside the blocks.
# MLXB_FOLD_NORMS=0 (or setting this to False before a model is loaded) keeps every norm a kernel of its own.
FOLD_NORMS = os.environ.get("MLXB_FOLD_NORMS", "1") != "0"


class PreNormBlock(Block):
    replayable = True
    kernel_libs = ("gemm_smallm_fold", "norm")     # what folding a norm into a linear layer launches from
    def __init__(self, norm_1: Norm, mixer: Mixer, norm_2: Norm, feed_forward: FeedForward):
        self.norm_1, self.mixer, self.norm_2, self.feed_forward = norm_1, mixer, norm_2, feed_forward
        self._defer_1 = self._defer_2 = False

    def children(self):
        return (self.norm_1, self.mixer, self.norm_2, self.feed_forward)

    def cache_spec(self):
        return self.mixer.cache_spec()

    def bind_all(self, tensors, dtype, device) -> None:
        super().bind_all(tensors, dtype, device)
        fold = FOLD_NORMS and dtype == torch.bfloat16
        self._defer_1 = fold and self.mixer.fold_input_norm(self.norm_1)
        self._defer_2 = fold and self.feed_forward.fold_input_norm(self.norm_2)

    def forward(self, ctx, x, cache):
        n1 = self.norm_1.deferred(ctx, x) if self._defer_1 else self.norm_1.forward(ctx, x)
        h = self.mixer.forward(ctx, n1, x, cache)
        n2 = self.norm_2.deferred(ctx, h) if self._defer_2 else self.norm_2.forward(ctx, h)
        return self.feed_forward.forward(ctx, n2, h)


class StreamBlock(Block):
    """A pre-norm block over a float32 residual stream: ``x += mixer(norm_1(x))``, then, if the layer has a
    feed-forward, ``x += feed_forward(norm_2(x))``, then any number of further branches, each of which reads the
    stream and adds to it (``branch.forward(ctx, x) -> x``).  Norms give the run's dtype to the products; the sums
    stay float32 whatever the run's dtype is."""
    replayable = True

    def __init__(self, norm_1: Norm, mixer: Mixer, norm_2: Optional[Norm] = None,
                 feed_forward: Optional[FeedForward] = None, branches=()):
        if (norm_2 is None) != (feed_forward is None):
            raise ValueError("a feed-forward and the norm before it come together")
        self.norm_1, self.mixer, self.norm_2, self.feed_forward = norm_1, mixer, norm_2, feed_forward
        self.branches = tuple(branches)

    def children(self):
        return tuple(p for p in (self.norm_1, self.mixer, self.norm_2, self.feed_forward) if p is not None) + self.branches

    def cache_spec(self):
        return self.mixer.cache_spec()

    def forward(self, ctx, x, cache):
        x = self.mixer.forward(ctx, self.norm_1.forward(ctx, x), x, cache)
        if self.feed_forward is not None:
            x = self.feed_forward.forward(ctx, self.norm_2.forward(ctx, x), x)
        for b in self.branches:
            x = b.forward(ctx, x)
        return x


class ParallelBlock(Block):
    """A block over a float32 residual stream whose two sublayers read the same normed input:
    ``h = norm_1(x); x += mixer(h) + feed_forward(h)``.  There is one norm; the feed-forward is optional.  Each
    sublayer adds its result to the stream itself (the mixer in its last product's epilogue)."""
    replayable = True

    def __init__(self, norm_1: Norm, mixer: Mixer, feed_forward: Optional[FeedForward] = None):
        self.norm_1, self.mixer, self.feed_forward = norm_1, mixer, feed_forward

    def children(self):
        return tuple(p for p in (self.norm_1, self.mixer, self.feed_forward) if p is not None)

    def cache_spec(self):
        return self.mixer.cache_spec()

    def forward(self, ctx, x, cache):
        h = self.norm_1.forward(ctx, x)
        x = self.mixer.forward(ctx, h, x, cache)
        if self.feed_forward is not None:
            x = self.feed_forward.forward(ctx, h, x)
        return x


class SandwichBlock(Block):
    """A block over a float32 residual stream with a norm before AND after each sublayer:
    ``x += post_1(mixer(norm_1(x)))``, then, if the layer has a feed-forward, ``x += post_2(feed_forward(norm_2(x)))``.

    The sublayers leave their results in float32 (``mixer.mix(ctx, x, cache) -> [T, width]``,
    ``feed_forward.branch(ctx, x) -> ([T * terms, width], terms)``: a feed-forward of experts hands over one row per
    (token, chosen expert), summed in the update).  The post-norms are elementwise (``Norm.stream_args()``), so one
    kernel does the sum over terms, the post-norm, the add to the stream and the norm that reads the stream next:
    ``norm_2`` of this block, or ``norm_1`` of the block named by ``feeds`` (the one that runs next), whose input
    then waits in ``ctx.carried``.  Norms in front that are not elementwise run as kernels of their own."""
    replayable = True
    kernel_libs = ("dyt",)

    def __init__(self, norm_1: Norm, mixer: Mixer, post_1: Norm, norm_2: Optional[Norm] = None,
                 feed_forward: Optional[FeedForward] = None, post_2: Optional[Norm] = None,
                 feeds: Optional["SandwichBlock"] = None):
        if not (norm_2 is None) == (feed_forward is None) == (post_2 is None):
            raise ValueError("a feed-forward comes with the norm before it and the norm after it")
        self.norm_1, self.mixer, self.post_1 = norm_1, mixer, post_1
        self.norm_2, self.feed_forward, self.post_2 = norm_2, feed_forward, post_2
        self.feeds = feeds

    def children(self):
        return tuple(p for p in (self.norm_1, self.mixer, self.post_1, self.norm_2, self.feed_forward, self.post_2)
                     if p is not None)

    def cache_spec(self):
        return self.mixer.cache_spec()

    @staticmethod
    def _fusable(norm: Optional[Norm]) -> bool:
        return norm is not None and hasattr(norm, "stream_args") and getattr(norm, "out_scale", 1.0) == 1.0

    def _update(self, ctx, x, branch, terms: int, post: Norm, nxt: Optional[Norm], tag: str, name: str):
        T, D = x.shape
        out = None
        if self._fusable(nxt):
            out = ctx.ws.get(tag, T, D, ctx.dtype)
        ops.label(name, (12.0 + terms) * T * D, (8.0 + 4.0 * terms + (out.element_size() if out is not None else 0)) * T * D)
        ops.dyt_residual(x, branch, ctx.stream, post=post.stream_args(), nxt=nxt.stream_args() if out is not None else None,
                         next_out=out, terms=terms, token_req=ctx.token_req)
        return out

    def forward(self, ctx, x, cache):
        carried = getattr(ctx, "carried", None)
        ctx.carried = None
        if carried is not None and carried[0] is self.norm_1:
            n1 = carried[1]
        else:
            n1 = self.norm_1.forward(ctx, x)
        y = self.mixer.mix(ctx, n1, cache)
        if self.feed_forward is None:
            nxt = self.feeds.norm_1 if self.feeds is not None else None
            out = self._update(ctx, x, y, 1, self.post_1, nxt, "normed", self.post_1.name)
            if out is not None:
                ctx.carried = (nxt, out)
            return x
        n2 = self._update(ctx, x, y, 1, self.post_1, self.norm_2, "normed_2", self.post_1.name)
        if n2 is None:
            n2 = self.norm_2.forward(ctx, x, tag="normed_2")
        yb, terms = self.feed_forward.branch(ctx, n2)
        nxt = self.feeds.norm_1 if self.feeds is not None else None
        out = self._update(ctx, x, yb, terms, self.post_2, nxt, "normed", self.post_2.name)
        if out is not None:
            ctx.carried = (nxt, out)
        return x


class HyperBlock(Block):
    """A pre-norm block over several float32 residual streams (hyper-connections), ``x`` being ``[x_1 | .. | x_S]``.  Around
    each sublayer ``q`` (1: the mixer, 2: the feed-forward, if the layer has one):
    ``y = sublayer(norm_q(sum_s in_q[s] x_s))``, then, all streams from the old ones,
    ``x_t <- sum_s mix_q[s, t] x_s + residual_scale * out_q[t] y`` (``<name>.hc<q>.in``, ``.out``, ``.mix``, float32).
    ``learned=False``: no such tensors; ``in``, ``out`` and ``mix`` are 1 (one stream: an ordinary residual sum with a factor).

    The sublayers leave their results in float32 (``mixer.mix``, ``feed_forward.branch`` with one row a token), and one
    kernel does the streams' update together with what reads them next: the weighted sum and the norm of this block's
    second sublayer, or of the block that runs next (``ctx.next_block``), whose input then waits in ``ctx.carried``.  The
    norms are RMS norms (``Norm.rms_args()``)."""
    replayable = True
    kernel_libs = ("streams",)

    def __init__(self, name: str, n_streams: int, norm_1: Norm, mixer: Mixer, norm_2: Optional[Norm] = None,
                 feed_forward: Optional[FeedForward] = None, residual_scale: float = 1.0, learned: bool = True):
        if (norm_2 is None) != (feed_forward is None):
            raise ValueError("a feed-forward and the norm before it come together")
        if not learned and n_streams != 1:
            raise ValueError(f"{name}: {n_streams} streams need tensors that say how they are read and mixed")
        if not 1 <= n_streams <= 16:
            raise ValueError(f"{name}: {n_streams} residual streams (1 to 16)")
        self.name, self.n_streams, self.residual_scale, self.learned = name, int(n_streams), float(residual_scale), learned
        self.norm_1, self.mixer, self.norm_2, self.feed_forward = norm_1, mixer, norm_2, feed_forward
        self.connections = {}          # sublayer -> (in, residual_scale * out, mix)

    def children(self):
        return tuple(p for p in (self.norm_1, self.mixer, self.norm_2, self.feed_forward) if p is not None)

    def cache_spec(self):
        return self.mixer.cache_spec()

    def _sublayers(self):
        return (1,) if self.feed_forward is None else (1, 2)

    def param_specs(self):
        S, specs = self.n_streams, []
        if self.learned:
            for q in self._sublayers():
                n = f"{self.name}.hc{q}"
                specs += [ParamSpec(n + ".in", (S,), VECTOR, Init(1.0 / S, 0.3 / S)), ParamSpec(n + ".out", (S,), VECTOR, Init(1.0, 0.2)),
                          ParamSpec(n + ".mix", (S, S), VECTOR, Init(1.0 / S, 0.3 / S))]
        return specs

    def bind(self, tensors, dtype, device) -> None:
        for q in self._sublayers():
            if self.learned:
                n = f"{self.name}.hc{q}"
                w_in, w_out, mix = (tensors[f"{n}.{t}"].contiguous() for t in ("in", "out", "mix"))
            else:
                w_in, w_out, mix = (torch.ones(s, dtype=torch.float32, device=device) for s in ((1,), (1,), (1, 1)))
            self.connections[q] = (w_in, w_out * self.residual_scale, mix)

    def _reader(self, q: int):
        norm = self.norm_1 if q == 1 else self.norm_2
        weight, eps = norm.rms_args()
        return norm, self.connections[q][0], weight, eps

    def _read(self, ctx, x):
        norm, w_in, weight, eps = self._reader(1)
        T, D = x.shape[0], norm.width
        out = ctx.ws.get("normed", T, D, ctx.dtype)
        ops.label(norm.name, (2.0 * self.n_streams + 4.0) * T * D, (4.0 * self.n_streams + out.element_size()) * T * D)
        ops.streams_read(x, self.n_streams, w_in, weight, out, eps, ctx.stream)
        return out

    def _update(self, ctx, x, y, q: int, reader, tag: str):
        T, D, S = y.shape[0], y.shape[1], self.n_streams
        _, w_out, mix = self.connections[q]
        out, kw = None, {}
        if reader is not None:
            _, w_in, weight, eps = reader
            out = ctx.ws.get(tag, T, D, ctx.dtype)
            kw = dict(nxt=(w_in, weight), next_out=out, eps=eps)
        ops.label(f"{self.name}.hc{q}", (2.0 * S * S + 4.0 * S + 4.0) * T * D,
                  (8.0 * S + 4.0 + (out.element_size() if out is not None else 0)) * T * D)
        ops.streams_update(x, y, S, mix, w_out, ctx.stream, token_req=ctx.token_req, **kw)
        return out

    def forward(self, ctx, x, cache):
        carried, ctx.carried = getattr(ctx, "carried", None), None
        n1 = carried[1] if carried is not None and carried[0] is self else self._read(ctx, x)
        nxt = getattr(ctx, "next_block", None)
        if not (isinstance(nxt, HyperBlock) and nxt.n_streams == self.n_streams):
            nxt = None
        y = self.mixer.mix(ctx, n1, cache)
        if self.feed_forward is not None:
            n2 = self._update(ctx, x, y, 1, self._reader(2), "normed_2")
            y, terms = self.feed_forward.branch(ctx, n2)
            if terms != 1:
                raise ops.KernelError(f"{self.name}: a feed-forward that leaves {terms} rows a token")
        out = self._update(ctx, x, y, 2 if self.feed_forward is not None else 1, nxt._reader(1) if nxt is not None else None,
                           "normed")
        if out is not None:
            ctx.carried = (nxt, out)
        return x


class OutputNormBlock(Block):
    """A block over a float32 residual stream with a norm on every sublayer's result and none before it:
    ``x += norm_1(mixer(x))``, then, if the layer has a feed-forward, ``x += norm_2(feed_forward(x))``.

    The sublayers read the stream itself (in the run's dtype) and leave their results in float32 (``mixer.mix``,
    ``feed_forward.summands``); one kernel adds a feed-forward's summands up, norms the sum (an RMS norm,
    ``Norm.rms_args()``), adds it to the stream and leaves the new rows in the run's dtype for what reads them next: this
    block's feed-forward, or the block that runs next (``ctx.next_block``), whose input then waits in ``ctx.carried``."""
    replayable = True
    kernel_libs = ("rms", "elementwise")

    def __init__(self, norm_1: Norm, mixer: Mixer, norm_2: Optional[Norm] = None, feed_forward: Optional[FeedForward] = None):
        if (norm_2 is None) != (feed_forward is None):
            raise ValueError("a feed-forward and the norm on its result come together")
        self.norm_1, self.mixer, self.norm_2, self.feed_forward = norm_1, mixer, norm_2, feed_forward

    def children(self):
        return tuple(p for p in (self.norm_1, self.mixer, self.norm_2, self.feed_forward) if p is not None)

    def cache_spec(self):
        return self.mixer.cache_spec()

    def _rows(self, ctx, x):
        """The stream's rows in the run's dtype."""
        if ctx.dtype == torch.float32:
            return x
        out = ctx.ws.get("stream_rows", *x.shape, ctx.dtype)
        ops.label("stream.cast", 0.0, (4.0 + out.element_size()) * x.numel())
        ops.join_rows(x, None, out, ctx.stream)
        return out

    def _update(self, ctx, x, y: Summands, norm: Norm, read_next: bool):
        """``x += norm(y)``; the new rows in the run's dtype where something reads them next."""
        T, D = x.shape
        cast = ctx.ws.get("stream_rows", T, D, ctx.dtype) if read_next and ctx.dtype != torch.float32 else None
        weight, eps = norm.rms_args()
        ops.label(norm.name, (6.0 + y.terms) * T * D, (8.0 + 4.0 * y.terms + (4.0 if y.extra is not None else 0.0)
                                                       + (cast.element_size() if cast is not None else 0.0)) * T * D)
        ops.norm_update(x, y.rows, weight, eps, ctx.stream, terms=y.terms, scale=y.scale, y2=y.extra, token_req=ctx.token_req,
                        cast_out=cast)
        return x if cast is None else cast

    def forward(self, ctx, x, cache):
        carried, ctx.carried = getattr(ctx, "carried", None), None
        h = carried[1] if carried is not None and carried[0] is self else self._rows(ctx, x)
        nxt = getattr(ctx, "next_block", None)
        if not isinstance(nxt, OutputNormBlock):
            nxt = None
        y = Summands(self.mixer.mix(ctx, h, cache))
        if self.feed_forward is None:
            h = self._update(ctx, x, y, self.norm_1, nxt is not None)
        else:
            h = self._update(ctx, x, y, self.norm_1, True)
            h = self._update(ctx, x, self.feed_forward.summands(ctx, h), self.norm_2, nxt is not None)
        if nxt is not None:
            ctx.carried = (nxt, h)
        return x


register_part("block", "output_norm", OutputNormBlock)
register_part("block", "hyper", HyperBlock)
register_part("block", "pre_norm", PreNormBlock)
register_part("block", "parallel", ParallelBlock)
register_part("block", "sandwich", SandwichBlock)
register_part("block", "stream", StreamBlock)

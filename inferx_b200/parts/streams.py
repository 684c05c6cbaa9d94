"""Several residual streams beside each other (hyper-connections).

The stream is fp32 [T, n, width].  ``StreamCopies`` (an embedding) starts all n copies from
the embedding table's row.  ``HyperConnection`` holds one sublayer's weights: what it reads,
u = sum_s read[s] x_s, and how its output y enters, x_t <- sum_s mix[s, t] x_s + put[t] y, all
streams at once from the old ones.  ``HyperConnectedBlock`` arranges a layer: a sublayer's
output stays pending (``StreamUpdate``) until the next reading, which applies the update,
forms u and norms it in one pass over the streams when the norm works entry by entry
(``forward_streams``); another norm gets u, written in fp32, and does the rest itself.  What a
mixture of experts leaves unwritten is combined in that same pass.
"""
from __future__ import annotations

from dataclasses import replace

import torch

from ..weights.loader import TensorDecl
from .base import StreamUpdate
from .registry import build_part, register_part


def read_streams(ops, norm, streams, update, read, rows=None):
    """What a sublayer sees: the streams after ``update`` (kept unless ``rows`` picks rows to
    gather), weighted by ``read`` and normed."""
    if hasattr(norm, "forward_streams"):
        return norm.forward_streams(streams, update, read, rows=rows)
    u = ops.stream_step(streams, update, read, None, torch.float32, rows=rows)
    return norm.forward(u, None)


class StreamCopies:
    """The embedding table's row in every stream."""

    def __init__(self, spec, ctx, prefix: str):
        self.spec, self.ctx, self.streams = spec, ctx, int(spec.streams)
        if self.streams < 1:
            raise ValueError(f"{prefix}: {spec.streams} residual streams")
        self.ones = torch.ones(self.streams, dtype=torch.float32, device=ctx.device)

    def check_limits(self):
        check = getattr(self.ctx.ops, "check_stream_limits", None)
        if check is not None:
            check(self.streams, "residual streams")

    def tensors(self):
        return []

    def bind(self, w):
        pass

    def cache_needs(self):
        return []

    def forward(self, embed_table, step, cache):
        return self.ctx.ops.embed_streams(embed_table, step.token_ids, self.streams)


class HyperConnection:
    """One sublayer's reading weights [n], writing weights [n] and mixing matrix [from, to]."""

    def __init__(self, spec, ctx, prefix: str, optional: bool = False):
        self.spec, self.prefix, self.optional = spec, prefix, optional
        self.read = self.put = self.mix = None

    def tensors(self):
        n = self.spec.streams
        r, p, m = (f"{self.prefix}.{x}" for x in self.spec.names)
        return [TensorDecl(r, (n,), keep="float32", init="gain", optional=self.optional),
                TensorDecl(p, (n,), keep="float32", init="gain", optional=self.optional),
                TensorDecl(m, (n, n), keep="float32", init="bias", optional=self.optional)]

    def bind(self, w):
        if self.optional:
            return
        self.read, self.put, self.mix = (w[f"{self.prefix}.{x}"].contiguous()
                                         for x in self.spec.names)


class _Unused:
    """Tensors of a sublayer that a layer has not: a checkpoint may hold them all the same."""

    def __init__(self, part):
        self.part = part

    def tensors(self):
        return [replace(d, optional=True) for d in self.part.tensors()]

    def bind(self, w):
        pass


class HyperConnectedBlock:
    """``u = read(x); y = sublayer(norm(u)); x <- mix(x) + put y`` for the mixer and then for
    the feed-forward, on several streams; a layer may have no feed-forward."""

    def __init__(self, spec, ctx, prefix: str):
        p = prefix
        self.spec, self.ctx = spec, ctx
        self.input_norm = build_part("norm", spec.input_norm, ctx, f"{p}.{spec.input_norm_name}")
        self.mixer = build_part("mixer", spec.mixer, ctx, f"{p}.{spec.mixer_name}")
        self.ffn = build_part("feed_forward", spec.ffn, ctx, f"{p}.{spec.ffn_name}")
        self.post_norm = build_part("norm", spec.post_norm, ctx, f"{p}.{spec.post_norm_name}")
        first, second = spec.connection.sublayers
        self.mixer_link = HyperConnection(spec.connection, ctx, f"{p}.{first}")
        self.ffn_link = HyperConnection(spec.connection, ctx, f"{p}.{second}",
                                        optional=self.ffn is None)

    def parts(self):
        own = [self.input_norm, self.mixer, self.mixer_link, self.ffn_link]
        if self.ffn is None:
            return own + [_Unused(self.post_norm)]
        return own + [self.post_norm, self.ffn]

    def cache_needs(self):
        return list(self.mixer.cache_needs())

    def forward(self, streams, pending, step, cache):
        ops = self.ctx.ops
        h = read_streams(ops, self.input_norm, streams, pending, self.mixer_link.read)
        link = self.mixer_link
        pending = StreamUpdate(self.mixer.forward(h, step, cache), link.mix, link.put)
        if self.ffn is None:
            return pending
        link = self.ffn_link
        h = read_streams(ops, self.post_norm, streams, pending, link.read)
        return StreamUpdate(self.ffn.forward(h, step), link.mix, link.put)


register_part("embedding", "stream_copies", StreamCopies)
register_part("block", "hyper_connected", HyperConnectedBlock)

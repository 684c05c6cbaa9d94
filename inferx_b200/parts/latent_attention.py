"""Latent attention: keys and values of all heads are widened from one small cached
vector per token.

Per token the input is projected down to ``kv_rank + rot_dim`` numbers: the first
``kv_rank``, RMS-normed, are the latent ``c``; the rest is a rotated key part shared by
all heads.  Head h's key is ``(W_uk[h] c | k_rot)`` and its value ``W_uv[h] c``; only
``c`` and ``k_rot`` are cached, as one record per token.  The key matrix is folded into
the query instead of widening cached latents:

    q_plain . (W_uk[h] c) = (W_uk[h]^T q_plain) . c

so attention runs with one shared key head of ``kv_rank + rot_dim`` entries whose values
are the latents themselves, and the head's output ``sum_j p_j c_j`` is widened by
``W_uv[h]`` afterwards.  Every step - a whole prompt, a portion, a decoded token - takes
this one path through the cache, so a position's result does not depend on how its
sequence was cut.  Queries carry ``dim`` plain and ``rot_dim`` rotated entries per head;
an optional sigmoid gate computed from the mixer's input multiplies the heads' outputs
before the output projection.

The projections that read the input (query, down-projection, gate) are one product over
concatenated weights; the per-head products are library calls batched over heads.

Two options.  Queries may go through a latent of their own (``q_rank``): the first product
then makes c_q beside the down-projection, one pass normalises c_q and writes the record,
and a second product widens c_q to the queries.  A layer without records of its own
(``own_records`` off) has no down-projection: the schedule points it at another layer's
cache, which holds that layer's records of this step too by the time it runs.
"""
from __future__ import annotations

import torch

from ..weights.loader import TensorDecl
from .base import PagedKvNeed
from .registry import build_part, register_part

ENTRY = "latent"


class LatentAttentionMixer:
    def __init__(self, spec, ctx, prefix: str):
        self.spec, self.ctx, self.prefix = spec, ctx, prefix
        self.position = build_part("position", spec.position, ctx, prefix)
        self.names = dict(spec.names)
        self.in_w = self.uk_t = self.uv = self.o_w = self.latent_gain = None
        s = spec
        self.q_width = s.heads * (s.dim + s.rot_dim)
        self.q_rank = s.q_rank              # -1 until the checkpoint says it
        self.uq_w = self.q_gain = None
        self._place()

    def _place(self):
        """Columns of the first product: query (or its latent), down-projection, gate."""
        s = self.spec
        self.kv_off = self.q_rank if self.q_rank else self.q_width
        self.gate_off = self.kv_off + (s.kv_rank + s.rot_dim if s.own_records else 0)

    def check_limits(self):
        check = getattr(self.ctx.ops, "check_latent_attention_limits", None)
        if check is not None:
            check(self.spec.kv_rank, self.spec.rot_dim, self.prefix)

    def _n(self, key):
        return f"{self.prefix}.{self.names[key]}"

    def tensors(self):
        s = self.spec
        hv = s.heads * s.vdim
        if s.q_rank:
            decls = [TensorDecl(self._n("dq"), (s.q_rank, s.hidden)),
                     TensorDecl(self._n("dq_norm"), (s.q_rank,), keep="float32", init="gain"),
                     TensorDecl(self._n("uq"), (self.q_width, s.q_rank))]
        else:
            decls = [TensorDecl(self._n("q"), (self.q_width, s.hidden))]
        if s.own_records:
            decls += [TensorDecl(self._n("dkv"), (s.kv_rank + s.rot_dim, s.hidden)),
                      TensorDecl(self._n("dkv_norm"), (s.kv_rank,), keep="float32",
                                 init="gain")]
        decls += [
            TensorDecl(self._n("uk"), (s.heads * s.dim, s.kv_rank)),
            TensorDecl(self._n("uv"), (hv, s.kv_rank)),
            TensorDecl(self._n("o"), (s.hidden, hv)),
        ]
        if s.output_gate:
            decls.append(TensorDecl(self._n("g"), (hv, s.hidden)))
        return decls

    def bind(self, w):
        s = self.spec
        parts = [w[self._n("dq" if s.q_rank else "q")]]
        if s.q_rank:
            self.uq_w, self.q_gain = w[self._n("uq")], w[self._n("dq_norm")]
            self.q_rank = self.uq_w.shape[1]
            if parts[0].shape[0] != self.q_rank or self.q_gain.numel() != self.q_rank:
                raise ValueError(f"{self.prefix}: {parts[0].shape[0]} rows make the query's "
                                 f"latent, {self.q_rank} columns read it")
        if s.own_records:
            parts.append(w[self._n("dkv")])
            self.latent_gain = w[self._n("dkv_norm")]
        if s.output_gate:
            parts.append(w[self._n("g")])
        self._place()
        self.in_w = torch.cat(parts, dim=0).contiguous()
        # [heads, kv_rank, dim]: q_lat[h] = q_plain[h] . uk[h] summed over dim
        self.uk_t = w[self._n("uk")].view(s.heads, s.dim, s.kv_rank).transpose(1, 2).contiguous()
        self.uv = w[self._n("uv")].view(s.heads, s.vdim, s.kv_rank).contiguous()
        self.o_w = w[self._n("o")]

    def cache_needs(self):
        s = self.spec
        if not s.own_records:
            return []
        return [PagedKvNeed(1, s.kv_rank + s.rot_dim, s.window, entries=(ENTRY,))]

    def _queries(self, x, proj, step, cache, group, records):
        """(rotated query parts, plain ones heads outermost); the step's records are in the
        cache when this returns."""
        s, ops = self.spec, self.ctx.ops
        if self.position is not None:
            freq, mag, rot_dims = self.position.pair_table()
        else:
            freq, mag, rot_dims = torch.empty(0, dtype=torch.float32, device=x.device), 1.0, 0
        writes = s.own_records and cache.writes
        if not s.q_rank and s.own_records:
            return ops.latent_prepare(
                proj, 0, self.kv_off, step.positions, freq, mag, self.latent_gain, s.latent_eps,
                s.heads, s.dim, s.rot_dim, rot_dims, s.kv_rank,
                records if writes else None, group.slots if writes else None)
        q = proj
        if s.q_rank:
            c_q = ops.latent_front(
                proj, self.q_rank, self.q_gain, s.latent_eps, self.kv_off, step.positions, freq,
                mag, self.latent_gain, s.kv_rank, s.rot_dim, rot_dims,
                records if writes else None, group.slots if writes else None)
            q = ops.linear(c_q, self.uq_w)
        return ops.latent_queries(q, step.positions, freq, mag, s.heads, s.dim, s.rot_dim,
                                  rot_dims)

    def forward(self, x, step, cache):
        s, ops = self.spec, self.ctx.ops
        T = x.shape[0]
        group = step.groups[cache.group]
        records = cache.pages[ENTRY]
        proj = ops.linear(x, self.in_w)
        q_rot, q_plain = self._queries(x, proj, step, cache, group, records)
        q_lat = ops.batched_linear(q_plain, self.uk_t)                       # [heads, T, rank]
        mixed = ops.latent_attention(q_lat, q_rot, records, group.block_table, step, s.window,
                                     s.scale, **({"fp32_weights": True} if s.fp32_weights
                                                 else {}))                   # [heads, T, rank]
        if s.output_gate:
            o = ops.gate_heads(ops.batched_linear(mixed, self.uv), proj, self.gate_off)
        else:
            # the heads' values land beside each other, ready for the output projection
            o = torch.empty((T, s.heads, s.vdim), dtype=x.dtype, device=x.device)
            ops.batched_linear(mixed, self.uv, out=o.transpose(0, 1))        # [heads, T, vdim]
            o = o.view(T, s.heads * s.vdim)
        return ops.linear(o, self.o_w, out_dtype=torch.float32 if s.out_float32 else None)


register_part("mixer", "latent_attention", LatentAttentionMixer)

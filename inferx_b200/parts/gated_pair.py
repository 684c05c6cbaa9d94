"""A gated recurrence without a matrix of state, and two mixers joined into one.

* ``MinGruMixer`` (kind "min_gru"): z = sigmoid(W_z h + b_z), u = W_x h + b_x, candidate
  c = u + shift where u >= 0 and sigmoid(u) below; entry by entry S_t = (1 - z) S_(t-1) +
  z c; the output is W_o (S_t * silu(W_g h)).  S lives in fp32 in the cache manager's state
  slots (zeroed when a slot is handed out) and the gates, the candidate and the walk are
  fp32.  Because the gates do not read S, a token is the affine map S -> (1 - z) S + z c and
  a long portion is walked in pieces side by side whose maps are joined.
* ``ScaledPairMixer`` (kind "scaled_pair"): left_scale * left + right_scale * right of two
  mixers that read the same input.  Two mixers that come in halves (``front_matrices``,
  ``mix_front``, ``out_matrix``: see ``DistanceAttentionMixer``) run as one: a single product
  makes everything either reads, each writes its result, times its scale, into its own
  columns of one row, and a single product over the two output matrices laid side by side
  adds them in its accumulators.  Any other two mixers run one after the other.
"""
from __future__ import annotations

import torch

from ..weights.loader import TensorDecl
from .base import StateNeed
from .registry import build_part, register_part

STATE = "min_gru_state"


class MinGruMixer:
    def __init__(self, spec, ctx, prefix: str):
        self.spec, self.ctx, self.prefix = spec, ctx, prefix
        self.front_width = 3 * spec.width
        self.inner = spec.width
        self.names = dict(spec.names)
        self.z_bias = self.x_bias = self.front_w = self.o_w = None

    def _n(self, key):
        return f"{self.prefix}.{self.names[key]}"

    def tensors(self):
        s = self.spec
        decls = [TensorDecl(self._n(k), (s.width, s.hidden)) for k in ("z", "x", "g")]
        decls += [TensorDecl(self._n(k), (s.width,), keep="float32", init="bias")
                  for k in ("z_bias", "x_bias")]
        return decls + [TensorDecl(self._n("o"), (s.hidden, s.width))]

    def front_matrices(self, w):
        return [w[self._n("z")], w[self._n("x")], w[self._n("g")]]

    def out_matrix(self, w):
        return w[self._n("o")]

    def bind_vectors(self, w):
        self.z_bias = w[self._n("z_bias")].contiguous()
        self.x_bias = w[self._n("x_bias")].contiguous()

    def bind(self, w):
        self.bind_vectors(w)
        self.front_w = torch.cat(self.front_matrices(w), dim=0).contiguous()
        self.o_w = self.out_matrix(w)

    def cache_needs(self):
        return [StateNeed(STATE, (self.spec.width,), torch.float32)]

    def mix_front(self, front, step, cache, out, out_scale):
        """``front`` [T, z | x | g] (a view of columns); ``out`` [T, width], a view too,
        receives S * silu(g) times ``out_scale``."""
        self.ctx.ops.min_gru(front, self.z_bias, self.x_bias, self.spec.shift,
                             cache.state[STATE], step, out, out_scale)

    def forward(self, x, step, cache):
        front = self.ctx.ops.linear(x, self.front_w)
        out = torch.empty((x.shape[0], self.inner), dtype=x.dtype, device=x.device)
        self.mix_front(front, step, cache, out, 1.0)
        return self.ctx.ops.linear(out, self.o_w)


class ScaledPairMixer:
    def __init__(self, spec, ctx, prefix: str):
        self.spec, self.ctx, self.prefix = spec, ctx, prefix
        self.left = build_part("mixer", spec.left, ctx, f"{prefix}.{spec.left_name}")
        self.right = build_part("mixer", spec.right, ctx, f"{prefix}.{spec.right_name}")
        self.joined = all(hasattr(m, "mix_front") for m in (self.left, self.right))
        self.front_w = self.out_w = None

    def check_limits(self):
        for m in (self.left, self.right):
            if hasattr(m, "check_limits"):
                m.check_limits()

    def tensors(self):
        return self.left.tensors() + self.right.tensors()

    def bind(self, w):
        if not self.joined:
            for m in (self.left, self.right):
                m.bind({d.name: w[d.name] for d in m.tensors()})
            return
        for m in (self.left, self.right):
            m.bind_vectors(w)
        self.front_w = torch.cat(self.left.front_matrices(w) + self.right.front_matrices(w),
                                 dim=0).contiguous()
        self.out_w = torch.cat([self.left.out_matrix(w), self.right.out_matrix(w)],
                               dim=1).contiguous()

    def cache_needs(self):
        return list(self.left.cache_needs()) + list(self.right.cache_needs())

    def forward(self, x, step, cache):
        s, ops, a, b = self.spec, self.ctx.ops, self.left, self.right
        if not self.joined:
            return (a.forward(x, step, cache).to(torch.float32) * s.left_scale
                    + b.forward(x, step, cache).to(torch.float32) * s.right_scale).to(x.dtype)
        front = ops.linear(x, self.front_w)
        both = torch.empty((x.shape[0], a.inner + b.inner), dtype=x.dtype, device=x.device)
        a.mix_front(front[:, :a.front_width], step, cache, both[:, :a.inner], s.left_scale)
        b.mix_front(front[:, a.front_width:], step, cache, both[:, a.inner:], s.right_scale)
        return ops.linear(both, self.out_w)


register_part("mixer", "min_gru", MinGruMixer)
register_part("mixer", "scaled_pair", ScaledPairMixer)

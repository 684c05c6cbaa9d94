"""A mixer with a matrix memory, exponential gates and a normaliser per head.

Per head, with the log gates i = cap tanh((W_i h + b_i) / cap) and f = logsigmoid(cap
tanh((W_f h + b_f) / cap)) and a running maximum m (0 before a sequence's first token):

    m_t = max(f + m_(t-1), i)
    S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T      (n likewise with k alone)
    o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + den_eps)

o is divided by its root mean square per head, multiplied by a gain over all heads and by
sigmoid(W_g h), and projected.  S, n and m are fp32 state per request in the cache manager's
slots, zeroed when a slot is handed out.  The gates, their running maximum, the memory and the
norm are fp32; the gates' projections leave their product in fp32.  The memory's kernels:
single tokens stream it through the chip once; portions of prompts are walked token by token,
or in chunks on the tensor cores where the sizes allow.
"""
from __future__ import annotations

import torch

from ..weights.loader import TensorDecl
from .base import StateNeed
from .registry import register_part

MEMORY, NORMALISER, MAXIMUM = "memory", "memory_normaliser", "memory_maximum"


def padded_rows(matrices, multiple: int = 8):
    """The matrices' rows one after the other, and zero rows up to a multiple: a product with
    them has rows on 16-byte marks."""
    w = torch.cat(list(matrices), dim=0)
    short = -w.shape[0] % multiple
    if short:
        w = torch.cat([w, torch.zeros((short, w.shape[1]), dtype=w.dtype, device=w.device)], dim=0)
    return w.contiguous()


class MatrixMemoryMixer:
    def __init__(self, spec, ctx, prefix: str):
        self.spec, self.ctx, self.p = spec, ctx, prefix
        self.hk, self.hv = spec.heads * spec.dim, spec.heads * spec.vdim

    def check_limits(self):
        check = getattr(self.ctx.ops, "check_matrix_memory_limits", None)
        if check is not None:
            check(self.spec.dim, self.p)

    def tensors(self):
        s, p = self.spec, self.p
        return [
            TensorDecl(f"{p}.q", (self.hk, s.hidden)), TensorDecl(f"{p}.k", (self.hk, s.hidden)),
            TensorDecl(f"{p}.v", (self.hv, s.hidden)), TensorDecl(f"{p}.g", (self.hv, s.hidden)),
            TensorDecl(f"{p}.o", (s.hidden, self.hv)),
            TensorDecl(f"{p}.norm", (self.hv,), keep="float32", init="gain"),
            TensorDecl(f"{p}.i", (s.heads, s.hidden)), TensorDecl(f"{p}.f", (s.heads, s.hidden)),
            TensorDecl(f"{p}.i.b", (s.heads,), keep="float32", init="bias"),
            TensorDecl(f"{p}.f.b", (s.heads,), keep="float32", init="bias"),
        ]

    def bind(self, w):
        p = self.p
        self.front_w = padded_rows([w[f"{p}.q"], w[f"{p}.k"], w[f"{p}.v"], w[f"{p}.g"]])
        self.gate_w = torch.cat([w[f"{p}.i"], w[f"{p}.f"]], dim=0).contiguous()
        self.gate_b = torch.cat([w[f"{p}.i.b"], w[f"{p}.f.b"]], dim=0).contiguous()
        self.norm_w, self.o_w = w[f"{p}.norm"], w[f"{p}.o"]

    def cache_needs(self):
        s = self.spec
        return [StateNeed(MEMORY, (s.heads, s.dim, s.vdim), torch.float32),
                StateNeed(NORMALISER, (s.heads, s.dim), torch.float32),
                StateNeed(MAXIMUM, (s.heads,), torch.float32)]

    def forward(self, x, step, cache):
        s, ops = self.spec, self.ctx.ops
        hk, hv = self.hk, self.hv
        gates = ops.memory_gates(x, self.gate_w, self.gate_b, s.gate_cap, cache.state[MAXIMUM],
                                 step)                       # fp32 [4, heads, T]
        front = ops.linear(x, self.front_w)                  # [T, q | k | v | g]
        y = ops.matrix_memory(
            front[:, :hk], front[:, hk:2 * hk], front[:, 2 * hk:2 * hk + hv], gates,
            cache.state[MEMORY], cache.state[NORMALISER], step, s.heads, s.dim, s.vdim, s.q_scale,
            finish=(self.norm_w, front[:, 2 * hk + hv:2 * hk + 2 * hv], s.norm_eps, s.den_eps))
        return ops.linear(y, self.o_w)


register_part("mixer", "matrix_memory", MatrixMemoryMixer)

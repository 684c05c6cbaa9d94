"""The Dominex design stated plainly, in float64, one function per mechanism.

Nothing here is shared with the engine: no part, no kernel face, no cache.  A model is a
``config`` (the parsed config.json) and ``weights`` (name -> tensor); ``forward`` runs a
whole sequence from position 0 and returns the logits of every position.  ``store`` is
applied wherever a run in a narrower element type would store an activation (the
identity by default; a rounding to bfloat16 imitates such a run, from which tests derive
their bounds).

Notation: h is a sublayer's input [T, width]; W x means x @ W.T for a stored [out, in];
eps is the configuration's norm.eps everywhere.
"""
from __future__ import annotations

import json
import math
import os

import torch

F64 = torch.float64


def read_model_folder(path):
    """(config.json as a dict, name -> tensor) of a model folder."""
    from inferx_b200.weights.safetensors_io import Checkpoint
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    ck = Checkpoint(path)
    w = {n: ck.get(n).clone() for n in ck.names()}
    ck.close()
    return cfg, w


def _w(weights, name):
    return weights[name].to(F64)


def ident(x):
    return x


def round_bf16(x):
    return x.to(torch.bfloat16).to(F64)


def round_f32(x):
    return x.to(torch.float32).to(F64)


# -- small functions ---------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_div(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    """The design's norm: the stored weight is the gain minus one."""
    return rms_div(x, eps) * (1.0 + w)


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


# -- attention in chunks with a distance penalty -------------------------------
def chunk_mask(n, size):
    """[n, n] bool: query i sees key j <= i when both lie in the same run of ``size``
    positions counted from 0 (size 0: every earlier key)."""
    i = torch.arange(n)
    vis = i[None, :] <= i[:, None]
    if size > 0:
        vis = vis & (i[:, None] // size == i[None, :] // size)
    return vis


def distance_penalty(n, r1, r2):
    """[heads, n, n]: r1_h ln(1 + r2_h (i - j)) for j <= i, zero elsewhere."""
    i = torch.arange(n, dtype=F64)
    d = torch.clamp(i[:, None] - i[None, :], min=0.0)
    return r1[:, None, None] * torch.log(1.0 + r2[:, None, None] * d[None])


def distance_attention(h, m, weights, p, store=ident):
    """Left mixer without its output projection: [T, heads * vdim]."""
    T = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = store(h @ _w(weights, f"{p}.q").T).view(T, H, dim)
    k = store(h @ _w(weights, f"{p}.k").T).view(T, G, dim)
    v = store(h @ _w(weights, f"{p}.v").T).view(T, G, vdim)
    own = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, own]) * m["scale"]
    s = s * _w(weights, f"{p}.temp")[:, None, None]
    s = s - distance_penalty(T, _w(weights, f"{p}.r1"), _w(weights, f"{p}.r2"))
    size = (m.get("mask") or {}).get("size", 0)
    s = s.masked_fill(~chunk_mask(T, size)[None], float("-inf"))
    a = torch.softmax(s, dim=-1)
    return torch.einsum("hij,jhd->ihd", a, v[:, own]).reshape(T, H * vdim)


# -- gated recurrence whose gates read the current token only ------------------
def gru_candidate(u):
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def min_gru_states(z, u, before=None):
    """S_t = (1 - z_t) S_(t-1) + z_t candidate(u_t), one row after another."""
    S = torch.zeros(z.shape[1], dtype=z.dtype) if before is None else before
    out = []
    for t in range(z.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * gru_candidate(u[t])
        out.append(S)
    return torch.stack(out)


def min_gru(h, weights, p, store=ident):
    """Right mixer without its output projection: [T, width of the state]."""
    z = sigmoid(store(h @ _w(weights, f"{p}.z").T) + _w(weights, f"{p}.z.b"))
    u = store(h @ _w(weights, f"{p}.x").T) + _w(weights, f"{p}.x.b")
    g = store(h @ _w(weights, f"{p}.g").T)
    return min_gru_states(z, u) * silu(g)


def parallel_mixer(h, m, weights, p, store=ident):
    a = store(distance_attention(h, m["left"], weights, f"{p}.left", store))
    b = store(min_gru(h, weights, f"{p}.right", store))
    return (m["left_scale"] * (a @ _w(weights, f"{p}.left.o").T)
            + m["right_scale"] * (b @ _w(weights, f"{p}.right.o").T))


# -- latent attention ------------------------------------------------------------
def rotate_neighbours(x, positions, base):
    """x [T, ..., d]: pair (2i, 2i+1) turned by position * base^(-2i/d)."""
    d = x.shape[-1]
    f = torch.tensor([float(base) ** (-2.0 * i / d) for i in range(d // 2)], dtype=F64)
    a = positions.to(F64).view(-1, *([1] * (x.dim() - 1))) * f
    u, v = x[..., 0::2], x[..., 1::2]
    out = torch.empty_like(x)
    out[..., 0::2] = u * torch.cos(a) - v * torch.sin(a)
    out[..., 1::2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def latent_records(h, m, weights, p, eps, positions, store=ident):
    """(latents [T, kv_rank], rotated key part [T, rot_dim]) of a layer with its own
    down-projection."""
    down = store(h @ _w(weights, f"{p}.dkv").T)
    r = m["kv_rank"]
    c = store(rms_div(down[:, :r], eps) * _w(weights, f"{p}.dkv.norm"))
    k_rot = store(rotate_neighbours(down[:, r:], positions, m["rot"]["base"]))
    return c, k_rot


def latent_attention(h, m, weights, p, eps, positions, records, store=ident):
    """The mixer on ``records`` (its own or another layer's), with output projection."""
    T = h.shape[0]
    H, dim, rot, vdim = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_rot = records
    cq = store(rms_div(store(h @ _w(weights, f"{p}.dq").T), eps) * _w(weights, f"{p}.dq.norm"))
    q = store(cq @ _w(weights, f"{p}.uq").T).view(T, H, dim + rot)
    q_rot = store(rotate_neighbours(q[..., dim:], positions, m["rot"]["base"]))
    k = store(c @ _w(weights, f"{p}.uk").T).view(T, H, dim)
    v = store(c @ _w(weights, f"{p}.uv").T).view(T, H, vdim)
    s = (torch.einsum("ihd,jhd->hij", q[..., :dim], k)
         + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    s = s.masked_fill(~chunk_mask(T, 0)[None], float("-inf"))
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v).reshape(T, H * vdim)
    return store(o) @ _w(weights, f"{p}.o").T


# -- mixture of experts -------------------------------------------------------------
def route(z, top):
    """(experts [T, top] by falling score, their scores, margin of the choice): scores are
    sigmoid(z); equal scores go to the lower index."""
    order = torch.sort(z, dim=-1, descending=True, stable=True).indices
    chosen = order[:, :top]
    s = sigmoid(z)
    w = torch.gather(s, 1, chosen)
    if top < z.shape[1]:
        margin = w[:, -1] - torch.gather(s, 1, order[:, top:top + 1])[:, 0]
    else:
        margin = torch.ones(z.shape[0], dtype=z.dtype)
    return chosen, w, margin


def expert(h, weights, p, store=ident):
    a = silu(h @ _w(weights, f"{p}.gate").T) * (h @ _w(weights, f"{p}.up").T)
    return store(store(a) @ _w(weights, f"{p}.down").T)


def mixture(h, f, weights, p, store=ident, margins=None):
    """Sum over the chosen experts of expert(score * h)."""
    chosen, w, margin = route(h @ _w(weights, f"{p}.router").T, f["router"]["top"])
    if margins is not None:
        for t in range(h.shape[0]):
            margins[t] = min(margins[t], float(margin[t]))
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        rows, slots = torch.nonzero(chosen == e, as_tuple=True)
        if rows.numel():
            out[rows] += expert(w[rows, slots][:, None] * h[rows], weights, f"{p}.e{e}", store)
    return out


# -- the whole model ------------------------------------------------------------------
def forward(cfg, weights, tokens, store=ident, layers_out=None, margins=None):
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    T = tokens.numel()
    positions = torch.arange(T)
    if margins is not None:
        margins.extend([math.inf] * T)
    table = _w(weights, "embed")
    x = table[tokens] * cfg["embedding"]["scale"]
    records = {}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}"
        h = store(norm_around_zero(x, _w(weights, f"{p}.norm1"), eps))
        if layer["type"] == "parallel":
            x = x + parallel_mixer(h, m, weights, f"{p}.mix", store)
        elif layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                records[i] = latent_records(h, m, weights, f"{p}.mix", eps, positions, store)
                src = i
            x = x + latent_attention(h, m, weights, f"{p}.mix", eps, positions, records[src],
                                     store)
        else:
            raise ValueError(layer["type"])
        if layer.get("mlp") is not None:
            h = store(norm_around_zero(x, _w(weights, f"{p}.norm2"), eps))
            x = x + mixture(h, layer["mlp"], weights, f"{p}.mlp", store, margins)
        if layers_out is not None:
            layers_out.append(x.clone())
    n = store(norm_around_zero(x, _w(weights, "final.norm"), eps))
    return softcap(n @ table.T, cfg["logit_softcap"])

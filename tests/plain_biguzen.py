"""The Biguzen design stated plainly, in float64, one function per mechanism.

Nothing here is shared with the engine: no part, no kernel face, no cache.  A model is a
``config`` (the parsed config.json) and ``weights`` (name -> tensor); ``forward`` runs a
whole sequence from position 0 and returns the logits of every position.  ``store`` is
applied wherever a run in a narrower element type would store an activation (the
identity by default; a rounding to bfloat16 imitates such a run, from which tests derive
their bounds).

Notation: h is a sublayer's input [T, width]; W x means x @ W.T for a stored [out, in];
eps is the configuration's norm.eps.
"""
from __future__ import annotations

import json
import math
import os

import torch
import torch.nn.functional as F

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


# -- norm --------------------------------------------------------------------------
def dynamic_tanh(x, alpha, w, b):
    """Entry by entry; nothing of the row enters."""
    return torch.tanh(alpha * x) * w + b


def model_norm(x, weights, name):
    return dynamic_tanh(x, _w(weights, f"{name}.alpha"), _w(weights, name),
                        _w(weights, f"{name}.b"))


def rms_div(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# -- several residual streams --------------------------------------------------------
def stream_read(streams, read):
    """streams [s, T, width], read [s]: what a sublayer's norm sees."""
    return sum(read[s] * streams[s] for s in range(streams.shape[0]))


def stream_update(streams, y, mix, write):
    """Every new stream t is sum_s mix[s, t] (old stream s) + write[t] * y."""
    n = streams.shape[0]
    return torch.stack([sum(mix[s, t] * streams[s] for s in range(n)) + write[t] * y
                        for t in range(n)])


# -- rotation --------------------------------------------------------------------------
def frequencies(dims, base, factor=1.0):
    return [base ** (-2.0 * i / dims) / factor for i in range(dims // 2)]


def rotate_pairs(x, positions, freqs, dims):
    """x [T, heads, dim]: neighbours (2i, 2i+1) of the first ``dims`` entries are turned by
    position * frequency."""
    if not dims:
        return x
    ang = torch.tensor(positions, dtype=F64)[:, None] * torch.tensor(freqs, dtype=F64)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# -- short convolution over time ---------------------------------------------------
def causal_conv(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before 0."""
    T, C = u.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=u.dtype), u], dim=0)
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


# -- attention ---------------------------------------------------------------------
def visible(T, size):
    """[T, T]: query i sees key j."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    ok = d >= 0
    return ok & (d < size) if size else ok


def attend(q, k, v, scale, size, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv].  ``sink`` [H]: exp(sink_h)
    joins the denominator of head h."""
    T, H, _ = q.shape
    G = k.shape[1]
    ok = visible(T, size)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = torch.where(ok, s, torch.tensor(-math.inf, dtype=F64))
        m = torch.maximum(s.max(-1, keepdim=True).values, sink[h])
        e = torch.exp(s - m)
        out[:, h] = (e / (e.sum(-1, keepdim=True) + torch.exp(sink[h] - m))) @ v[:, g]
    return out


def attention(h, weights, p, m, positions, kept, store=ident):
    """The mixer "attention".  ``kept``: None, or (keys, values) of the layer it reads in
    the place of its own.  Returns (output, keys, values)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m.get("vdim", m["dim"])

    def project(n, heads, size):
        u = store(h @ _w(weights, f"{p}.{n}").T + _w(weights, f"{p}.{n}.b"))
        if m.get("conv", 0):
            u = store(causal_conv(u, _w(weights, f"{p}.{n}.conv")))
        return u.reshape(T, heads, size)

    rot = m.get("rot")
    dims, freqs = 0, []
    if rot:
        dims = rot["dims"]
        freqs = frequencies(dims, rot["base"], (rot.get("scaling") or {}).get("factor", 1.0))
    q = store(rotate_pairs(project("q", H, d), positions, freqs, dims))
    if kept is None:
        k = store(rotate_pairs(project("k", G, d), positions, freqs, dims))
        v = project("v", G, dv)
    else:
        k, v = kept
    o = attend(q, k, v, m["scale"], (m.get("mask") or {}).get("size", 0),
               _w(weights, f"{p}.sink"))
    gate = torch.sigmoid(store(h @ _w(weights, f"{p}.g").T))
    o = store(store(o) * gate[:, :, None]).reshape(T, H * dv)
    return o @ _w(weights, f"{p}.o").T, k, v


# -- matrix memory -----------------------------------------------------------------------
def log_gates(h, weights, p, cap):
    """(log input gate, log forget gate), each [T, heads]."""
    zi = h @ _w(weights, f"{p}.i").T + _w(weights, f"{p}.i.b")
    zf = h @ _w(weights, f"{p}.f").T + _w(weights, f"{p}.f.b")
    return cap * torch.tanh(zi / cap), F.logsigmoid(cap * torch.tanh(zf / cap))


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, dv], log gates [T, H] -> o [T, H, dv], token by token."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64)
    n = torch.zeros(H, d, dtype=F64)
    m = torch.zeros(H, dtype=F64)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hd,hdv->hv", q[t], S) / den[:, None]
    return out


def mlstm(h, weights, p, m, eps, store=ident):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m.get("vdim", m["dim"])
    q = store(h @ _w(weights, f"{p}.q").T).reshape(T, H, d) * d ** -0.5
    k = store(h @ _w(weights, f"{p}.k").T).reshape(T, H, d)
    v = store(h @ _w(weights, f"{p}.v").T).reshape(T, H, dv)
    i, f = log_gates(h, weights, p, m["gate_cap"])
    o = rms_div(matrix_memory(q, k, v, i, f), eps).reshape(T, H * dv)
    gate = torch.sigmoid(store(h @ _w(weights, f"{p}.g").T))
    return store(o * _w(weights, f"{p}.norm") * gate) @ _w(weights, f"{p}.o").T


# -- feed-forward --------------------------------------------------------------------
def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def two_matrices(h, weights, p, act, store=ident):
    return store(act(store(h @ _w(weights, f"{p}.up").T))) @ _w(weights, f"{p}.down").T


def group_values(pick, count):
    """A group's value: the sum of its two largest choice scores."""
    size = pick.numel() // count
    return [float(pick[g * size:(g + 1) * size].sort(descending=True).values[:2].sum())
            for g in range(count)]


def choose(scores, correction, top, group_count, group_keep, scale):
    """scores [n] = sigmoid of the router's outputs.  Returns (indices, weights)."""
    n = scores.numel()
    pick = scores + correction
    size = n // group_count
    value = group_values(pick, group_count)
    kept = sorted(range(group_count), key=lambda g: (-value[g], g))[:group_keep]
    allowed = [e for e in range(n) if e // size in kept]
    idx = sorted(allowed, key=lambda e: (-float(pick[e]), e))[:top]
    w = scores[idx]
    return idx, w / (w.sum() + 1e-20) * scale


def choice_margin(scores, correction, top, group_count, group_keep):
    """How far the choice is from another one: the smaller of the distance between the last
    kept group and the first one left out and that between the last chosen expert and the
    first one left out (infinite where nothing is left out)."""
    n = scores.numel()
    pick = scores + correction
    size = n // group_count
    value = group_values(pick, group_count)
    order = sorted(range(group_count), key=lambda g: (-value[g], g))
    margin = math.inf
    if group_keep < group_count:
        margin = value[order[group_keep - 1]] - value[order[group_keep]]
    kept = order[:group_keep]
    allowed = sorted((float(pick[e]) for e in range(n) if e // size in kept), reverse=True)
    if top < len(allowed):
        margin = min(margin, allowed[top - 1] - allowed[top])
    return margin


def moe_ff(h, weights, p, f, store=ident, margins=None):
    r = f["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    scores = torch.sigmoid(h @ _w(weights, f"{p}.router").T)
    corr = _w(weights, f"{p}.correction")
    per_token = torch.zeros(h.shape[0], r["experts"], dtype=F64)
    for t in range(h.shape[0]):
        idx, w = choose(scores[t], corr, r["top"], groups["count"], groups["keep"],
                        r.get("scale", 1.0))
        per_token[t, idx] = w
        if margins is not None:
            margins[t] = min(margins[t], choice_margin(scores[t], corr, r["top"],
                                                       groups["count"], groups["keep"]))
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        rows = (per_token[:, e] != 0).nonzero()[:, 0]
        if rows.numel():
            out[rows] += per_token[rows, e, None] * two_matrices(h[rows], weights, f"{p}.e{e}",
                                                                 gelu_erf, store)
    if f.get("shared"):
        gate = torch.sigmoid(h @ _w(weights, f"{p}.shared.sg").T)
        out = out + gate * two_matrices(h, weights, f"{p}.shared", gelu_erf, store)
    return out


# -- the model -----------------------------------------------------------------------
def forward(cfg, weights, tokens, store=ident, layers_out=None, margins=None):
    """Logits [T, vocab].  ``layers_out`` (a list) receives the sum of the streams after
    every layer; ``margins`` (a list) receives, per token, the smallest ``choice_margin``
    of its routers."""
    eps = cfg["norm"]["eps"]
    if margins is not None:
        margins[:] = [math.inf] * len(tokens)
    positions = list(range(len(tokens)))
    x = _w(weights, "embed")[torch.tensor(tokens)]
    streams = torch.stack([x] * cfg["streams"])
    held = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", layer["mixer"], layer.get("mlp")

        def sublayer(q, run):
            h = store(model_norm(stream_read(streams, _w(weights, f"{p}.hc{q}.in")), weights,
                                 f"{p}.norm{q}"))
            return stream_update(streams, store(run(h)), _w(weights, f"{p}.hc{q}.mix"),
                                 _w(weights, f"{p}.hc{q}.out"))

        def mix(h):
            if layer["type"] == "mlstm":
                return mlstm(h, weights, f"{p}.mix", m, eps, store)
            src = m.get("kv_from")
            out, k, v = attention(h, weights, f"{p}.mix", m, positions,
                                  None if src is None else held[src], store)
            if src is None:
                held[i] = (k, v)
            return out

        streams = sublayer(1, mix)
        if f is not None and f["kind"] == "dense":
            streams = sublayer(2, lambda h: two_matrices(h, weights, f"{p}.mlp", relu_squared,
                                                         store))
        elif f is not None:
            streams = sublayer(2, lambda h: moe_ff(h, weights, f"{p}.mlp", f, store, margins))
        if layers_out is not None:
            layers_out.append(streams.sum(0))
    h = store(model_norm(streams.sum(0), weights, "final.norm"))
    return h @ _w(weights, "embed").T

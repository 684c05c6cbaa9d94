"""Shared pieces of the Biguzen tests: small configurations, model folders, the plain
model's rows and the error bounds."""
import random

import torch

import plain_biguzen as plain
from inferx_b200.weights.random_model import write_random_model


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale=None, groups=None, shared=0):
    router = {"experts": experts, "top": top}
    if scale is not None:
        router["scale"] = scale
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def memory(heads, dim, vdim, cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": mlp}


def attention(heads, kv_heads, dim, vdim, scale, window, conv=0, rot=None, kv_from=None, mlp=None):
    """rot = (dims, base, factor or None); window 0: every earlier key."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if conv:
        m["conv"] = conv
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if rot[2] is not None:
            m["rot"]["scaling"] = {"factor": rot[2]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def top(vocab, width, streams, eps, layers):
    return {"architecture": "Biguzen", "vocab": vocab, "width": width, "streams": streams,
            "norm": {"eps": eps}, "layers": layers}


# odd sizes, nothing a multiple of 8; five streams; a reader whose window is wider than that of
# the layer whose keys it reads, and one with a narrower one; convolutions of five taps, of one
# and none; no window, no rotation; no groups, no shared expert; a layer without feed-forward
BA = top(101, 60, 5, 1e-5, [
    memory(3, 10, 6, 4.0, mlp=dense(33)),
    attention(5, 1, 6, 10, 0.6, 5, conv=5, rot=(4, 50.0, None), mlp=moe(5, 2, 18, scale=0.7)),
    attention(5, 1, 6, 10, 0.5, 9, conv=1, rot=(4, 50.0, None), kv_from=1, mlp=dense(25)),
    attention(3, 3, 10, 7, 0.4, 0),
    attention(5, 1, 6, 10, 0.45, 2, rot=(4, 50.0, None), kv_from=1, mlp=moe(3, 3, 12)),
    memory(1, 7, 12, 9.0, mlp=moe(6, 1, 20, groups=(3, 1), shared=10)),
])

# three streams; groups of two and of four; a shared expert; the reader follows its source
# after a layer between; wide value heads; factors on the frequencies
BB = top(211, 96, 3, 1e-6, [
    attention(6, 2, 24, 40, 0.3, 11, conv=3, rot=(12, 300.0, 4.0),
              mlp=moe(8, 3, 24, scale=1.7, groups=(4, 2), shared=40)),
    memory(4, 16, 24, 15.0, mlp=moe(8, 2, 16, scale=2.0, groups=(2, 1))),
    attention(6, 2, 24, 40, 0.25, 7, conv=2, rot=(12, 300.0, 4.0), kv_from=0, mlp=dense(72)),
    memory(2, 24, 8, 6.0),
])

# sizes of the kind a served model has: heads the tensor-core kernels take, two streams
BC = top(512, 256, 2, 1e-5, [
    memory(4, 64, 64, 12.0, mlp=dense(384)),
    attention(8, 2, 64, 64, 0.125, 48, conv=4, rot=(32, 10000.0, 2.0),
              mlp=moe(8, 8, 128, scale=1.2, shared=128)),
    attention(8, 2, 64, 64, 0.11, 100, conv=4, rot=(32, 10000.0, 2.0), kv_from=1,
              mlp=moe(4, 4, 64)),
    memory(2, 32, 128, 20.0, mlp=dense(256)),
    attention(4, 1, 128, 128, 0.08, 40, conv=2, rot=(128, 1000.0, None), mlp=dense(128)),
])

# one stream; memories alone (no pages at all)
BD = top(67, 40, 1, 1e-6, [
    memory(2, 20, 12, 8.0, mlp=dense(56)),
    memory(5, 8, 8, 3.0, mlp=moe(4, 2, 24, groups=(2, 2), shared=16)),
])

CONFIGS = {"BA": BA, "BB": BB, "BC": BC, "BD": BD}


def sharpen(name, t):
    """N(0, 0.02) weights would give uniform attention, memories that hold next to nothing,
    routers without an opinion, streams that are copies of one another and gates at a half;
    make each of them matter."""
    last = name.rsplit(".", 1)[-1]
    if name == "embed":
        return t * 40.0
    if ".hc" in name:
        if last == "mix":
            return t * 15.0 + torch.eye(t.shape[0])
        return (t - 1.0) * 20.0 + (1.0 / t.shape[0] if last == "in" else 1.0)
    if name.endswith(".alpha"):
        return t * 0.6
    if name.endswith(".f.b"):
        return t * 25.0 + 2.0
    if name.endswith(".i.b"):
        return t * 25.0
    if name.endswith((".mix.q", ".mix.k")):
        return t * 6.0
    if name.endswith((".mix.v", ".mix.i", ".mix.f", ".mix.g", ".shared.sg")):
        return t * 5.0
    if name.endswith(".conv"):
        return t * 25.0
    if name.endswith(".sink"):
        return t * 60.0
    if name.endswith(".router"):
        return t * 12.0
    if name.endswith(".correction"):
        return t * 25.0
    if name.endswith(".b"):
        return t * 15.0
    if name.endswith((".up", ".down")):
        return t * 3.0
    return t


def make_model_dir(cfg, path, seed, dtype="float32", adjust=sharpen):
    write_random_model(cfg, str(path), seed=seed, dtype=dtype, adjust=adjust)
    return str(path)


def make_requests(cfg, lengths, seed):
    rng = random.Random(seed)
    return {f"r{i}": [rng.randrange(cfg["vocab"]) for _ in range(n)]
            for i, n in enumerate(lengths)}


def reference_rows(model_dir, requests):
    cfg, w = plain.read_model_folder(model_dir)
    rows = {}
    for rid, toks in requests.items():
        lg = plain.forward(cfg, w, toks).to(torch.float32)
        for p in range(len(toks)):
            rows[(rid, p)] = lg[p]
    return rows


def _bound(model_dir, requests, store, factor, floor):
    cfg, w = plain.read_model_folder(model_dir)
    worst = 0.0
    for toks in requests.values():
        a = plain.forward(cfg, w, toks)
        b = plain.forward(cfg, w, toks, store=store)
        worst = max(worst, float((a - b).abs().max()) / float(a.abs().max()))
    return max(floor, factor * worst)


def bound_for(dtype, model_dir, requests):
    """Three times what storing activations in the run's element type costs the plain
    model itself, relative to the largest logit; the floors stand for sums of hundreds of
    products in that precision, which the plain model does not have."""
    if dtype == "float32":
        return _bound(model_dir, requests, plain.round_f32, 3.0, 3e-5)
    return _bound(model_dir, requests, plain.round_bf16, 3.0, 5e-3)


def decisive_rows(model_dir, requests, least=5e-3):
    """{(request, position)} whose logits cannot have been changed by a router's close
    call: no router of this or an earlier token of the request chose with a margin below
    ``least``, neither in the plain model nor in the plain model that rounds what it stores
    to bfloat16 (a choice that rounding can turn changes the token's streams, and through
    keys, values and memories every later token's).  Tests of bfloat16 runs compare these
    rows; the 32-bit runs compare all."""
    cfg, w = plain.read_model_folder(model_dir)
    keep = set()
    for rid, toks in requests.items():
        exact, rounded = [], []
        plain.forward(cfg, w, toks, margins=exact)
        plain.forward(cfg, w, toks, store=plain.round_bf16, margins=rounded)
        for p, (a, b) in enumerate(zip(exact, rounded)):
            if min(a, b) < least:
                break
            keep.add((rid, p))
    return keep


def rows_to_compare(dtype, model_dir, requests, rows, share=0.1):
    """The produced rows a run in ``dtype`` is held to (see ``decisive_rows``)."""
    if dtype == "float32":
        return rows
    keep = decisive_rows(model_dir, requests)
    kept = {k: v for k, v in rows.items() if k in keep}
    assert len(kept) >= share * len(rows), "too many close calls: the test compares too little"
    return kept

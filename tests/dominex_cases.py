"""Shared pieces of the Dominex tests: small configurations, model folders, the plain
model's rows and the error bounds."""
import random

import torch

import plain_dominex as plain
from inferx_b200.weights.random_model import write_random_model


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def parallel(heads, kv_heads, dim, vdim, scale, chunk, width, scales, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk:
        left["mask"] = {"size": chunk}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left, "right": {"width": width}, "left_scale": scales[0],
                      "right_scale": scales[1]}}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
         "q_rank": q_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def top(vocab, width, scale, eps, cap, layers):
    return {"architecture": "Dominex", "vocab": vocab, "width": width,
            "embedding": {"scale": scale}, "norm": {"eps": eps}, "logit_softcap": cap,
            "layers": layers}


# two latent sources, one read twice and across other layers; value heads smaller and larger
# than key heads; chunks that are no multiple of a page; layers without a feed-forward
DA = top(197, 72, 3.0, 1e-6, 12.0, [
    latent(3, 12, 8, 20, 24, 28, 0.24, 700.0, mlp=moe(5, 2, 40)),
    parallel(6, 2, 16, 24, 0.25, 13, 56, (0.7, 1.3), mlp=moe(3, 3, 24)),
    latent(2, 8, 8, 12, 24, 20, 0.3, 700.0, kv_from=0, mlp=moe(4, 1, 32)),
    latent(4, 16, 4, 8, 40, 36, 0.22, 90.0),
    parallel(4, 1, 24, 16, 0.2, 21, 88, (1.1, 0.4)),
    latent(5, 20, 4, 16, 40, 44, 0.21, 90.0, kv_from=3, mlp=moe(6, 3, 16)),
    latent(3, 4, 8, 28, 24, 12, 0.29, 700.0, kv_from=0, mlp=moe(2, 1, 48)),
])

# odd sizes, nothing a multiple of 8; one head; chunks of one position, of two, none; as many
# key/value heads as heads; scales of one and a negative one
DB = top(89, 45, 1.0, 1e-5, 7.5, [
    parallel(1, 1, 7, 9, 0.4, 2, 31, (1.0, 1.0), mlp=moe(3, 2, 21)),
    parallel(5, 5, 6, 5, 0.4, 0, 13, (-0.6, 0.9), mlp=moe(2, 2, 10)),
    latent(1, 5, 2, 3, 11, 9, 0.37, 30.0, mlp=moe(4, 4, 9)),
    parallel(3, 1, 10, 6, 0.32, 1, 70, (0.5, 2.0)),
    latent(3, 3, 6, 7, 10, 13, 0.33, 10.0),
])

# sizes of the kind a served model has: the tensor-core kernels apply.  Only one layer leaves
# experts out, so that most rows of a bfloat16 run are free of close calls
def _served(choice):
    return top(512, 256, 16.0, 1e-5, 30.0, [
        parallel(8, 2, 64, 64, 0.125, 48, 256, (0.9, 1.2), mlp=moe(3, 3, 128)),
        latent(4, 32, 16, 48, 128, 112, 0.144, 10000.0, mlp=choice),
        latent(8, 48, 16, 32, 128, 160, 0.125, 10000.0, kv_from=1, mlp=moe(2, 2, 64)),
        parallel(4, 4, 128, 128, 0.088, 96, 320, (1.0, 0.8), mlp=moe(1, 1, 128)),
        parallel(16, 1, 64, 128, 0.12, 33, 192, (0.8, 1.0), mlp=moe(3, 3, 64)),
        latent(16, 64, 32, 64, 64, 104, 0.1, 500.0, mlp=moe(2, 2, 160)),
    ])


DC = _served(moe(6, 2, 96))
# the same without a choice at all: bfloat16 runs of hundreds of tokens compare every row
DD = _served(moe(4, 4, 96))

CONFIGS = {"DA": DA, "DB": DB, "DC": DC, "DD": DD}


def sharpen(name, t):
    """N(0, 0.02) weights would give uniform attention, gates of one half, routers without an
    opinion and penalties that are all alike; make each of them matter."""
    if name == "embed":
        return t * 25.0
    if name.endswith((".left.q", ".left.k", ".uk")):
        return t * 6.0
    if name.endswith((".dq", ".uq", ".dkv")):
        return t * 7.0
    if name.endswith((".v", ".uv", ".left.o", ".right.o", ".mix.o")):
        return t * 5.0
    if name.endswith((".right.z", ".right.x", ".right.g")):
        return t * 8.0
    if name.endswith((".z.b", ".x.b")):
        return t * 30.0
    if name.endswith((".norm1", ".norm2", "final.norm")):
        return t * 8.0
    if name.endswith(".r1"):
        return (t - 1.0) * 25.0 + 0.7
    if name.endswith(".r2"):
        return ((t - 1.0) * 12.0 + 0.4).abs()
    if name.endswith(".temp"):
        return (t - 1.0) * 15.0 + 1.3
    if name.endswith(".router"):
        return t * 10.0
    if name.endswith((".gate", ".up")):
        return t * 8.0
    if name.endswith(".down"):
        return t * 4.0
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


def decisive_rows(model_dir, requests, least=2e-3):
    """{(request, position)} whose logits cannot have been changed by a router's close
    call: no router of this or an earlier token of the request chose with a margin below
    ``least``, neither in the plain model nor in the plain model that rounds what it stores
    to bfloat16.  Tests of bfloat16 runs compare these rows; the 32-bit runs compare all."""
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


def rows_to_compare(dtype, model_dir, requests, rows, share=0.2):
    """The produced rows a run in ``dtype`` is held to (see ``decisive_rows``)."""
    if dtype == "float32":
        return rows
    keep = decisive_rows(model_dir, requests)
    kept = {k: v for k, v in rows.items() if k in keep}
    assert len(kept) >= share * len(rows), "too many close calls: the test compares too little"
    return kept

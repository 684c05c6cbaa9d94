"""Dominex configurations drawn at random: every size, count, order of layers and constant at
once, replayed against the plain model.  32-bit runs choose among experts; bfloat16 runs
choose all of them, so that no close call of a router can excuse a row."""
import random

import pytest

import dominex_cases as dk
import model_cases as mc
import traces
from inferx_b200.engine.replay import ReplaySession

pytestmark = pytest.mark.gpu


def draw(seed, choose):
    r = random.Random(seed)
    step = r.choice([1, 2, 8, 16])            # what the sizes are multiples of

    def size(lo, hi):
        return max(1, r.randint(lo, hi) // step) * step

    def mlp():
        if r.random() < 0.2:
            return None
        e = r.randint(1, 9 if choose else 4)
        return dk.moe(e, r.randint(1, e) if choose else e, size(8, 96))
    tensor = r.random() < 0.5                 # head sizes the tensor-core kernels take
    base, layers, sources = r.choice([30.0, 1000.0, 1e5]), [], []
    for i in range(r.randint(2, 6)):
        if r.random() < 0.5:
            g = r.choice([1, 1, 2, 3])
            dim, vdim = ((r.choice([64, 128]), r.choice([64, 128])) if tensor
                         else (size(3, 48), size(3, 48)))
            layers.append(dk.parallel(
                g * r.choice([1, 2, 4, 9]), g, dim, vdim, r.uniform(0.5, 1.5) * dim ** -0.5,
                r.choice([0, 1, 2, 7, 16, 31, 64, 90, 500]), size(5, 200),
                (r.uniform(-1.5, 1.5), r.uniform(0.2, 1.5)), mlp()))
            continue
        dim, heads, q_rank = size(2, 64), r.choice([1, 2, 3, 5, 8, 20]), size(4, 120)
        src = r.choice(sources) if sources and r.random() < 0.5 else None
        if src is None:
            rank = r.choice([64, 128, 256]) if tensor else size(5, 80)
            rot = r.choice([16, 32]) if tensor else 2 * r.randint(1, 12)
        else:
            rank, rot = layers[src]["mixer"]["kv_rank"], layers[src]["mixer"]["rot_dim"]
        layers.append(dk.latent(heads, dim, rot, size(2, 64), rank, q_rank,
                                r.uniform(0.5, 1.5) * (dim + rot) ** -0.5, base, src, mlp()))
        if src is None:
            sources.append(i)
    return dk.top(r.randint(40, 400), size(20, 200), r.uniform(0.5, 12.0), r.choice([1e-6, 1e-5]),
                  r.uniform(5.0, 40.0), layers), r


@pytest.mark.parametrize("seed", range(14))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_drawn_configuration(tmp_path, dtype, seed):
    cfg, r = draw(seed if dtype == "float32" else 100 + seed, dtype == "float32")
    d = dk.make_model_dir(cfg, tmp_path / "m", seed, dtype=dtype)
    reqs = dk.make_requests(cfg, [r.randint(1, 150) for _ in range(4)], seed)
    ref = dk.reference_rows(d, reqs)
    bound = dk.bound_for(dtype, d, reqs)
    for kind in ("whole", "tail", "portions", "mixed"):
        steps = mc.TRACE_KINDS[kind](reqs)
        sess = ReplaySession(d, dtype, traces.peak_tokens(steps), page_size=r.choice([4, 8, 16, 64]),
                             max_live=4)
        rows = mc.run_trace(sess, steps)
        sess.executor.poll_errors()
        mc.compare(rows, ref, bound, f"{seed}/{kind}/{dtype}")

"""Biguzen configurations drawn at random: every size, count, order of layers and constant at
once, replayed against the plain model.  32-bit runs choose among experts; bfloat16 runs
choose all of them, so that no close call of a router can excuse a row."""
import random

import pytest

import biguzen_cases as bk
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
        kind = r.random()
        if kind < 0.15:
            return None
        if kind < 0.4:
            return bk.dense(size(8, 200))
        groups = None
        if choose and r.random() < 0.7:
            count, per = r.choice([1, 2, 3, 4, 7]), r.choice([1, 2, 3, 5])
            keep = r.randint(1, count)
            e, top, groups = count * per, r.randint(1, keep * per), (count, keep)
        else:
            e = r.randint(1, 9 if choose else 4)
            top = r.randint(1, e) if choose else e
        return bk.moe(e, top, size(8, 96), scale=r.choice([None, 0.5, 2.5]), groups=groups,
                      shared=r.choice([0, size(8, 80)]))
    tensor = r.random() < 0.5                 # head sizes the tensor-core kernels take
    layers, sources = [], []
    for i in range(r.randint(2, 7)):
        if r.random() < 0.4:
            k, v = (16 * r.randint(1, 8), 8 * r.randint(1, 20)) if tensor else (size(3, 80), size(3, 80))
            layers.append(bk.memory(r.choice([1, 2, 3, 5]), k, v, r.uniform(2.0, 30.0), mlp()))
            continue
        window, conv = r.choice([0, 1, 2, 7, 16, 31, 64, 90, 500]), r.choice([0, 1, 2, 3, 4, 5, 9])
        if sources and r.random() < 0.5:
            src = r.choice(sources)
            m = layers[src]["mixer"]
            rot = m.get("rot")
            if rot is not None:
                rot = (rot["dims"], rot["base"], (rot.get("scaling") or {}).get("factor"))
            g, dim, vdim = m["kv_heads"], m["dim"], m["vdim"]
        else:
            src = None
            g = r.choice([1, 1, 2, 3])
            dim, vdim = ((r.choice([64, 128]), r.choice([64, 128])) if tensor
                         else (size(3, 48), size(3, 48)))
            rot = None
            if r.random() < 0.8 and dim >= 2:
                rot = (2 * r.randint(1, dim // 2), r.choice([30.0, 1000.0, 1e5]),
                       r.choice([None, 2.0, 7.5]))
            sources.append(i)
        heads = g * r.choice([1, 2, 4, 9])
        layers.append(bk.attention(heads, g, dim, vdim, r.uniform(0.5, 1.5) * dim ** -0.5, window,
                                   conv, rot, src, mlp()))
    return bk.top(r.randint(40, 400), size(20, 200), r.choice([1, 2, 3, 4, 6, 9]),
                  r.choice([1e-6, 1e-5]), layers), r


@pytest.mark.parametrize("seed", range(16))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_drawn_configuration(tmp_path, dtype, seed):
    cfg, r = draw(seed if dtype == "float32" else 100 + seed, dtype == "float32")
    d = bk.make_model_dir(cfg, tmp_path / "m", seed, dtype=dtype)
    reqs = bk.make_requests(cfg, [r.randint(1, 150) for _ in range(4)], seed)
    ref = bk.reference_rows(d, reqs)
    bound = bk.bound_for(dtype, d, reqs)
    for kind in ("whole", "tail", "portions", "mixed"):
        steps = mc.TRACE_KINDS[kind](reqs)
        sess = ReplaySession(d, dtype, traces.peak_tokens(steps), page_size=r.choice([4, 8, 16, 64]),
                             max_live=4)
        rows = mc.run_trace(sess, steps)
        sess.executor.poll_errors()
        mc.compare(rows, ref, bound, f"{seed}/{kind}/{dtype}")

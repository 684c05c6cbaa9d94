"""The Dominex design on the CPU: its configuration reader, the plain statement's own
mechanisms on values computed by hand, and the engine's host logic (pages of a run of
positions given back as the sequence leaves it, a layer that reads another layer's records,
the recurrence's state slots, batching) with the kernels replaced by their plain statements
(tests/host_ops.py)."""
import copy
import math

import pytest
import torch

import dominex_cases as dk
import host_ops
import model_cases as mc
import plain_dominex as plain
import traces
from inferx_b200.cache.manager import CacheGroup, CacheManager, groups_for
from inferx_b200.config.model_config import ConfigError
from inferx_b200.config.registry import config_from_json
from inferx_b200.engine.replay import ReplaySession

CASES = [("DA", dk.DA, 0, [5, 9, 27, 44, 3, 60], 4), ("DB", dk.DB, 1, [1, 6, 13, 31, 45], 8),
         ("DC", dk.DC, 3, [21, 1, 50, 2, 110], 16)]
D = torch.float64


# -- configuration ---------------------------------------------------------------
def test_config_reads_every_size_and_constant():
    cfg, spec = config_from_json(dk.DA)
    assert (cfg.vocab, cfg.width, cfg.embedding_scale, cfg.norm_eps, cfg.logit_softcap) == \
        (197, 72, 3.0, 1e-6, 12.0)
    assert (spec.embed_scale, spec.logit_softcap, spec.tied_head, spec.logit_scale) == \
        (3.0, 12.0, True, 1.0)
    assert (spec.final_norm.gain_offset, spec.final_norm.eps) == (1.0, 1e-6)
    a, b, c = (spec.layers[i].mixer for i in range(3))
    assert (a.kind, a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank, a.scale, a.window) == \
        ("latent_attention", 3, 12, 8, 20, 24, 28, 0.24, 0)
    assert a.own_records and not c.own_records and not a.output_gate
    assert (a.position.kind, a.position.rotary_dim, a.position.theta) == \
        ("rope_interleaved", 8, 700.0)
    assert (b.kind, b.left_scale, b.right_scale) == ("scaled_pair", 0.7, 1.3)
    assert (b.left.heads, b.left.kv_heads, b.left.head_dim, b.left.value_dim, b.left.scale,
            b.left.chunk) == (6, 2, 16, 24, 0.25, 13)
    assert (b.right.width, b.right.shift) == (56, 0.5)
    f = spec.layers[0].ffn
    assert (f.num_experts, f.top_k, f.expert_intermediate, f.score, f.weight_input,
            f.renormalize, f.shared) == (5, 2, 40, "sigmoid", True, False, None)
    assert spec.layers[3].ffn is None and spec.layers[3].post_norm is None
    assert [e.cache_of for e in spec.schedule] == [None, None, 0, None, None, 3, 0]
    again, _ = config_from_json(cfg.to_json())
    assert again == cfg


def test_config_without_optional_parts():
    obj = copy.deepcopy(dk.DB)
    obj.pop("embedding")
    obj.pop("logit_softcap")
    m = obj["layers"][0]["mixer"]
    m["left"].pop("mask")
    m["left"].pop("kv_heads")
    m["left"].pop("vdim")
    m.pop("left_scale")
    m.pop("right_scale")
    lat = obj["layers"][2]["mixer"]
    lat.pop("q_rank")
    lat.pop("rot")
    cfg, spec = config_from_json(obj)
    left = cfg.layers[0].pair.left
    assert (left.chunk, left.kv_heads, left.vdim) == (0, left.heads, left.dim)
    assert (cfg.layers[0].pair.left_scale, cfg.layers[0].pair.right_scale) == (1.0, 1.0)
    assert cfg.embedding_scale == 1.0 and spec.logit_softcap == 0.0
    assert spec.layers[2].mixer.q_rank == -1 and spec.layers[2].mixer.position is None


def _set(path, value):
    def change(obj):
        for k in path[:-1]:
            obj = obj[k]
        obj[path[-1]] = value
    return change


@pytest.mark.parametrize("change,match", [
    (_set(["layers", 1, "mixer", "left", "kv_heads"], 4), "key/value"),
    (_set(["layers", 1, "mixer", "left", "mask", "size"], -1), "mask.size"),
    (_set(["layers", 1, "type"], "pair"), "unknown layer type"),
    (_set(["layers", 0, "mlp", "kind"], "dense"), "unknown kind"),
    (_set(["layers", 0, "mlp", "router", "top"], 6), "of 5 experts"),
    (_set(["layers", 2, "mixer", "kv_from"], 1), "kv_from"),
    (_set(["layers", 6, "mixer", "kv_from"], 2), "kv_from"),
    (_set(["layers", 2, "mixer", "kv_from"], 2), "kv_from"),
    (_set(["layers", 2, "mixer", "kv_rank"], 25), "other sizes"),
    (_set(["layers", 2, "mixer", "rot", "base"], 701.0), "rotation"),
    (_set(["layers", 0, "mixer", "rot", "dims"], 7), "rot.dims"),
    (_set(["layers", 0, "mixer", "scale"], "big"), "scale"),
    (_set(["norm", "eps"], 0.0), "norm.eps"),
])
def test_config_refuses_what_it_cannot_run(change, match):
    obj = copy.deepcopy(dk.DA)
    change(obj)
    with pytest.raises(ConfigError, match=match):
        config_from_json(obj)


# -- the plain statement's mechanisms, by hand -----------------------------------------
def test_plain_norm_around_zero():
    x = torch.tensor([[3.0, 4.0]], dtype=D)
    got = plain.norm_around_zero(x, torch.tensor([0.0, 1.0], dtype=D), 0.5)
    r = math.sqrt(12.5 + 0.5)
    assert torch.allclose(got, torch.tensor([[3.0 / r, 8.0 / r]], dtype=D))


def test_plain_chunks_and_distance_by_hand():
    m = plain.chunk_mask(5, 2)
    assert m.tolist() == [[True, False, False, False, False], [True, True, False, False, False],
                          [False, False, True, False, False], [False, False, True, True, False],
                          [False, False, False, False, True]]
    assert torch.equal(plain.chunk_mask(4, 0), torch.tril(torch.ones(4, 4)).bool())
    p = plain.distance_penalty(3, torch.tensor([2.0, -1.0], dtype=D),
                               torch.tensor([0.5, 3.0], dtype=D))
    assert abs(p[0, 2, 0] - 2.0 * math.log(2.0)) < 1e-12 and p[0, 2, 2] == 0
    assert abs(p[1, 1, 0] + math.log(4.0)) < 1e-12


def test_plain_recurrence_by_hand():
    u = torch.tensor([[0.0], [-2.0], [1.5]], dtype=D)
    c = plain.gru_candidate(u)
    assert torch.allclose(c[:, 0], torch.tensor([0.5, 1 / (1 + math.exp(2.0)), 2.0], dtype=D))
    z = torch.tensor([[0.25], [0.5], [1.0]], dtype=D)
    s = plain.min_gru_states(z, u)[:, 0]
    s0 = 0.25 * 0.5
    s1 = 0.5 * s0 + 0.5 / (1 + math.exp(2.0))
    assert torch.allclose(s, torch.tensor([s0, s1, 2.0], dtype=D))


def test_plain_rotation_turns_neighbours():
    x = torch.tensor([[1.0, 0.0, 0.0, 2.0]], dtype=D)
    y = plain.rotate_neighbours(x, torch.tensor([3]), 100.0)[0]
    a0, a1 = 3.0, 3.0 / 10.0
    want = torch.tensor([math.cos(a0), math.sin(a0), -2 * math.sin(a1), 2 * math.cos(a1)], dtype=D)
    assert torch.allclose(y, want)


def test_plain_route_and_weight_on_the_input():
    z = torch.tensor([[0.0, 2.0, -1.0, 2.0]], dtype=D)
    e, w, margin = plain.route(z, 2)
    assert e.tolist() == [[1, 3]]
    s = 1 / (1 + math.exp(-2.0))
    assert torch.allclose(w, torch.tensor([[s, s]], dtype=D)) and abs(margin[0] - (s - 0.5)) < 1e-12
    # expert(w h) is not w expert(h)
    h = torch.tensor([[1.0, -2.0]], dtype=D)
    wt = {"p.router": torch.tensor([[2.0, 0.0], [-9.0, 0.0]], dtype=D),
          "p.e0.gate": torch.tensor([[1.0, 1.0]], dtype=D),
          "p.e0.up": torch.tensor([[3.0, 0.0]], dtype=D),
          "p.e0.down": torch.tensor([[1.0], [0.5]], dtype=D)}
    wt.update({k.replace("e0", "e1"): v for k, v in list(wt.items()) if "e0" in k})
    got = plain.mixture(h, {"router": {"experts": 2, "top": 1}}, wt, "p")
    g, u = s * -1.0, s * 3.0
    a = g / (1 + math.exp(-g)) * u
    assert torch.allclose(got, torch.tensor([[a, 0.5 * a]], dtype=D))


# -- the cache manager gives back the pages before a run -----------------------------------
def test_pages_before_the_run_at_hand_are_given_back():
    mgr = CacheManager([CacheGroup(chunk=10, layers=(0,)), CacheGroup(layers=(1,))], 16, 4, 2)
    mgr.open("a")
    assert mgr.reserve("a", 19)
    mgr.advance("a", 19)           # the next query sits at 19, in the run 10..19
    held = [p >= 0 for p in mgr.table("a", 0)]
    assert held == [False, False, True, True, True]      # positions 8..11 share a page
    assert all(p >= 0 for p in mgr.table("a", 1))
    mgr.check_invariants()
    assert mgr.reserve("a", 20)
    mgr.advance("a", 1)            # the next query starts the run at 20: everything goes
    assert [p >= 0 for p in mgr.table("a", 0)] == [False] * 5
    mgr.check_invariants()
    assert mgr.reserve("a", 24)
    mgr.advance("a", 4)
    assert [p >= 0 for p in mgr.table("a", 0)] == [False] * 5 + [True]
    mgr.close("a")
    assert mgr.free_pages(0) == 16 and mgr.free_pages(1) == 16


def test_groups_and_caches_of_the_layers():
    from inferx_b200.engine.runtime import Runtime, load_model
    from inferx_b200.weights.loader import RandomSource
    _, model = load_model(config_json=dk.DA, source=RandomSource(1), device="cpu",
                          dtype="float32", ops=host_ops)
    needs = model.cache_needs()
    spans = [(g.window, g.keep_first, g.chunk, g.layers) for g in groups_for(needs)]
    assert spans == [(0, 0, 0, (0, 3)), (0, 0, 13, (1,)), (0, 0, 21, (4,))]
    assert needs[2] == [] and needs[5] == [] and needs[6] == []      # they keep nothing
    rt = Runtime(model, page_size=4, num_pages=8, max_slots=2)
    caches = rt.executor.caches
    for reader, source in ((2, 0), (5, 3), (6, 0)):
        assert caches[reader].pages["latent"] is caches[source].pages["latent"]
        assert not caches[reader].writes and caches[source].writes
    assert rt.storage.state[1]["min_gru_state"].shape == (2, 56)
    assert rt.storage.state[1]["min_gru_state"].dtype == torch.float32


# -- the engine's host logic ---------------------------------------------------------
@pytest.mark.parametrize("name,cfg,seed,lengths,page", CASES)
@pytest.mark.parametrize("kind", list(mc.TRACE_KINDS))
def test_replay_matches_plain(tmp_path, name, cfg, seed, lengths, page, kind):
    d = dk.make_model_dir(cfg, tmp_path / "m", seed)
    reqs = dk.make_requests(cfg, lengths, seed)
    ref = dk.reference_rows(d, reqs)
    steps = mc.TRACE_KINDS[kind](reqs)
    sess = ReplaySession(d, "float32", traces.peak_tokens(steps), page_size=page, max_live=4,
                         device="cpu", ops=host_ops)
    rows = mc.run_trace(sess, steps)
    mc.compare(rows, ref, 3e-5, f"{name}/{kind}")
    if kind in ("whole", "tail", "portions"):
        assert len(rows) == sum(lengths)


def test_portions_of_two_tokens_and_single_tokens_agree_with_whole(tmp_path):
    d = dk.make_model_dir(dk.DB, tmp_path / "m", 7)
    toks = dk.make_requests(dk.DB, [27], 3)["r0"]
    ref = dk.reference_rows(d, {"a": toks})
    for size in (2, 1, 3, 5):
        steps = [{"step": i, "entries": [{"id": "a", "tokens": toks[a:a + size],
                                          "want": list(range(len(toks[a:a + size])))}],
                  "end": ["a"] if a + size >= len(toks) else []}
                 for i, a in enumerate(range(0, len(toks), size))]
        sess = ReplaySession(d, "float32", 64, page_size=4, max_live=1, device="cpu",
                             ops=host_ops)
        rows = mc.run_trace(sess, steps)
        assert len(rows) == len(toks)
        mc.compare(rows, ref, 3e-5, f"portions of {size}")


def test_state_slot_of_a_finished_request_starts_anew(tmp_path):
    d = dk.make_model_dir(dk.DA, tmp_path / "m", 2)
    reqs = dk.make_requests(dk.DA, [12, 9, 30], 5)
    ref = dk.reference_rows(d, reqs)
    sess = ReplaySession(d, "float32", 64, page_size=4, max_live=1, device="cpu", ops=host_ops)
    rows = mc.run_trace(sess, traces.whole(reqs))
    mc.compare(rows, ref, 3e-5, "slot reuse")


def test_a_mixer_beside_one_that_comes_whole(tmp_path):
    """A pair joins two mixers that come in halves and runs any other two one after the
    other, with the same result."""
    from inferx_b200.parts.base import BuildContext
    from inferx_b200.parts.gated_pair import ScaledPairMixer
    from inferx_b200.parts.specs import MinGruSpec, ScaledPairSpec
    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"), ops=host_ops)
    spec = ScaledPairSpec(hidden=12, left=MinGruSpec(12, 8), right=MinGruSpec(12, 5, shift=0.25),
                          left_scale=0.6, right_scale=-1.5)
    g = torch.Generator().manual_seed(3)
    mixers = [ScaledPairMixer(spec, ctx, "m") for _ in range(2)]
    w = {d.name: torch.randn(d.shape, generator=g) for d in mixers[0].tensors()}
    mixers[1].joined = False
    x = torch.randn(7, 12, generator=g)
    outs = []
    for m in mixers:
        m.bind(w)

        class step:
            cu_q = torch.tensor([0, 3, 7], dtype=torch.int32)
            state_slot = torch.tensor([1, 0], dtype=torch.int32)

        class half:
            state = None

        # the two recurrences keep a state under the same name: give each a cache of its own
        left, right = half(), half()
        left.state, right.state = {"min_gru_state": torch.zeros(2, 8)}, \
            {"min_gru_state": torch.zeros(2, 5)}
        lf, rf = m.left.mix_front, m.right.mix_front
        m.left.mix_front = lambda f, s, c, o, k, fn=lf, ca=left: fn(f, s, ca, o, k)
        m.right.mix_front = lambda f, s, c, o, k, fn=rf, ca=right: fn(f, s, ca, o, k)
        outs.append(m.forward(x, step, None))
    assert torch.allclose(outs[0], outs[1], atol=1e-5)


def test_greedy_generation_through_the_engine(tmp_path):
    from inferx_b200 import Engine, EngineConfig, Request, SamplingParams
    d = dk.make_model_dir(dk.DB, tmp_path / "m", 4)
    c, w = plain.read_model_folder(d)
    prompts = list(dk.make_requests(dk.DB, [7, 19, 3], 8).values())
    eng = Engine.create(EngineConfig(model=d, dtype="float32", device="cpu", block_size=4,
                                     max_num_seqs=2, num_gpu_blocks_override=64,
                                     prefill_chunk=5, max_model_len=64), ops=host_ops)
    done = eng.generate([Request(p, SamplingParams(max_tokens=6, ignore_eos=True))
                         for p in prompts])
    for p, c_out in zip(prompts, done):
        seq = list(p)
        for _ in range(6):
            seq.append(int(plain.forward(c, w, seq)[-1].argmax()))
        assert c_out.output_tokens == seq[len(p):]


def test_preemption_rebuilds_state_and_cache(tmp_path):
    """A pool too small for all three requests: the preempted ones give back pages and
    slot, start again from position 0, and generate the same tokens."""
    from inferx_b200 import Engine, EngineConfig, Request, SamplingParams
    d = dk.make_model_dir(dk.DA, tmp_path / "m", 0)
    reqs = dk.make_requests(dk.DA, [5, 9, 17], 0)

    def run(pages):
        eng = Engine.create(EngineConfig(model=d, dtype="float32", device="cpu", block_size=4,
                                         max_num_seqs=3, num_gpu_blocks_override=pages,
                                         max_model_len=64), ops=host_ops)
        outs = eng.generate([Request(t, SamplingParams(max_tokens=8, ignore_eos=True))
                             for t in reqs.values()])
        return [c.output_tokens for c in outs], eng.stats()["preemptions"]
    roomy, p0 = run(64)
    tight, p1 = run(6)
    assert p0 == 0 and p1 >= 1 and roomy == tight


def test_query_latent_size_comes_from_the_checkpoint(tmp_path):
    """A configuration may leave the size of the queries' latent to the tensors."""
    import json
    import os
    d = dk.make_model_dir(dk.DB, tmp_path / "m", 5)
    reqs = dk.make_requests(dk.DB, [9, 14], 1)
    ref = dk.reference_rows(d, reqs)
    path = os.path.join(d, "config.json")
    with open(path) as f:
        obj = json.load(f)
    for layer in obj["layers"]:
        layer["mixer"].pop("q_rank", None)
    with open(path, "w") as f:
        json.dump(obj, f)
    sess = ReplaySession(d, "float32", 128, page_size=4, max_live=2, device="cpu", ops=host_ops)
    mc.compare(mc.run_trace(sess, traces.whole(reqs)), ref, 3e-5, "size from the tensors")

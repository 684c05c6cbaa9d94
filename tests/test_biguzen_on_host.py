"""The Biguzen design on the CPU: its configuration reader, the plain statement's own
mechanisms on values computed by hand, and the engine's host logic (streams through the
schedule, memories and the convolutions' inputs in state slots, one layer's pages read by
others over windows of their own, batching) with the kernels replaced by their plain
statements (tests/host_ops.py)."""
import copy
import math
import os

import pytest
import torch

import biguzen_cases as bk
import host_ops
import model_cases as mc
import plain_biguzen as plain
import traces
from inferx_b200.cache.manager import groups_for
from inferx_b200.config.model_config import ConfigError
from inferx_b200.config.registry import config_from_json
from inferx_b200.engine.replay import ReplaySession

CASES = [("BA", bk.BA, 0, [5, 9, 17, 40, 3], 4), ("BB", bk.BB, 1, [1, 6, 13, 31, 45], 8),
         ("BD", bk.BD, 3, [21, 1, 40, 2, 27], 16)]
D = torch.float64


# -- configuration ---------------------------------------------------------------
def test_config_reads_every_size_and_constant():
    cfg, spec = config_from_json(bk.BA)
    assert (cfg.vocab, cfg.width, cfg.streams, cfg.norm_eps) == (101, 60, 5, 1e-5)
    assert spec.embedding.streams == 5 and spec.tied_head and spec.head_name == "embed"
    assert all(l.kind == "hyper_connected" and l.connection.streams == 5 for l in spec.layers)
    m = [l.mixer for l in spec.layers]
    assert (m[0].heads, m[0].dim, m[0].vdim, m[0].gate_cap, m[0].norm_eps, m[0].den_eps) == \
        (3, 10, 6, 4.0, 1e-5, 1e-6) and m[0].q_scale == 10 ** -0.5
    a = m[1]
    assert (a.heads, a.kv_heads, a.head_dim, a.value_dim, a.scale, a.window, a.conv_taps) == \
        (5, 1, 6, 10, 0.6, 5, 5)
    assert a.bias and a.learned_sink and a.head_gate and a.own_kv
    assert (a.position.layout, a.position.rotary_dim, a.position.theta, a.position.scaling) == \
        ("interleaved", 4, 50.0, None)
    # the pages of a layer are kept for the widest window among its readers
    assert a.cache_window == 9 and m[3].cache_window == 0
    assert [x.own_kv for x in m[1:5]] == [True, False, True, False]
    assert [e.cache_of for e in spec.schedule] == [None, None, 1, None, 1, None]
    f = [l.ffn for l in spec.layers]
    assert (f[0].kind, f[0].intermediate, f[0].activation) == ("mlp_activated", 33, "relu_squared")
    assert (f[1].num_experts, f[1].top_k, f[1].expert_intermediate, f[1].routed_scale, f[1].shared,
            f[1].group_count) == (5, 2, 18, 0.7, None, 0)
    assert (f[5].group_count, f[5].group_keep, f[5].group_value, f[5].renorm_eps, f[5].score,
            f[5].expert_activation, f[5].shared.intermediate, f[5].shared.activation) == \
        (3, 1, "pair_sum", 1e-20, "sigmoid", "gelu", 10, "gelu")
    assert f[3] is None
    again, _ = config_from_json(cfg.to_json())
    assert again == cfg
    _, spec = config_from_json(bk.BB)
    assert spec.layers[0].mixer.position.scaling == ("linear", 4.0)
    assert spec.layers[0].ffn.routed_scale == 1.7


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0].update(type="slstm"), "unknown layer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "unknown kind"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "key/value heads"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3), "rotated entries"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8), "rotated entries"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(scaling={"factor": 0}), "factor"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=-1), "must not be negative"),
    (lambda c: c["layers"][1]["mixer"].update(conv=-2), "must not be negative"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=3), "other sizes"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(base=51.0), "another rotation"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=3), "not an earlier attention layer"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=0), "not an earlier attention layer"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=4), "not an earlier attention layer"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "not an earlier attention layer"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=8), "other sizes"),
    (lambda c: c["layers"][0]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"].pop("gate_cap"), "'gate_cap' is missing"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=6), "of 5 experts"),
    (lambda c: c["layers"][5]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][5]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(heads="5"), "must be an integer"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "'scale' is missing"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.pop("width"), "'width' is missing"),
    (lambda c: c.update(layers=[]), "non-empty list"),
])
def test_config_refuses_what_it_cannot_run(change, match):
    cfg = copy.deepcopy(bk.BA)
    change(cfg)
    with pytest.raises(ConfigError, match=match):
        config_from_json(cfg)


# -- the plain statement's mechanisms ----------------------------------------------
def test_plain_norm_and_streams_by_hand():
    x = torch.tensor([[0.5, -2.0]], dtype=D)
    y = plain.dynamic_tanh(x, 0.5, torch.tensor([2.0, 3.0], dtype=D), torch.tensor([0.1, -0.2], dtype=D))
    assert torch.allclose(y, torch.tensor([[2 * math.tanh(0.25) + 0.1, 3 * math.tanh(-1.0) - 0.2]],
                                          dtype=D))
    s = torch.tensor([[[1.0]], [[10.0]]], dtype=D)             # two streams, one token
    assert float(plain.stream_read(s, torch.tensor([2.0, 3.0], dtype=D))) == 32.0
    mix = torch.tensor([[1.0, 5.0], [0.0, 2.0]], dtype=D)      # [from, to]
    out = plain.stream_update(s, torch.tensor([[7.0]], dtype=D), mix, torch.tensor([0.0, 1.0], dtype=D))
    assert out[:, 0, 0].tolist() == [1.0, 5.0 + 20.0 + 7.0]


def test_plain_memory_by_hand():
    """Two tokens, one head, one key entry, one value entry."""
    t = lambda *v: torch.tensor(v, dtype=D)
    q, k, v = t(2.0, 3.0).view(2, 1, 1), t(1.0, -4.0).view(2, 1, 1), t(5.0, 6.0).view(2, 1, 1)
    i, f = t(1.5, -2.0).view(2, 1), t(-0.5, -0.1).view(2, 1)
    out = plain.matrix_memory(q, k, v, i, f)
    m1 = max(-0.5 + 0.0, 1.5)                                  # the maximum starts at zero
    S1, n1 = math.exp(1.5 - m1) * 5.0, math.exp(1.5 - m1) * 1.0
    o1 = S1 * 2.0 / (max(abs(n1 * 2.0), math.exp(-m1)) + 1e-6)
    m2 = max(-0.1 + m1, -2.0)
    keep, put = math.exp(-0.1 + m1 - m2), math.exp(-2.0 - m2)
    S2, n2 = keep * S1 + put * -4.0 * 6.0, keep * n1 + put * -4.0
    o2 = S2 * 3.0 / (max(abs(n2 * 3.0), math.exp(-m2)) + 1e-6)
    assert torch.allclose(out.view(-1), t(o1, o2))
    # with weak input gates the maximum stays below zero's decay and the floor exp(-m) rules
    out = plain.matrix_memory(q, k, v, i - 9.0, f)
    m1 = max(-0.5, 1.5 - 9.0)
    S1 = math.exp(-7.5 - m1) * 5.0
    assert math.isclose(float(out[0]), S1 * 2.0 / (math.exp(-m1) + 1e-6))


def test_plain_gates_are_squashed():
    w = {"m.i": torch.ones(1, 1, dtype=D), "m.f": torch.ones(1, 1, dtype=D),
         "m.i.b": torch.tensor([1.0], dtype=D), "m.f.b": torch.tensor([-1.0], dtype=D)}
    i, f = plain.log_gates(torch.tensor([[100.0], [0.5]], dtype=D), w, "m", 4.0)
    assert abs(float(i[0]) - 4.0) < 1e-9 and math.isclose(float(i[1]), 4 * math.tanh(1.5 / 4))
    z = 4 * math.tanh(-0.5 / 4)
    assert math.isclose(float(f[1]), -math.log(1 + math.exp(-z)))


def test_plain_window_sink_rotation_and_convolution():
    ok = plain.visible(9, 3)
    assert [j for j in range(9) if ok[8, j]] == [6, 7, 8] and bool(plain.visible(9, 0)[8, 0])
    # scores of zero: weights 1 / (n + exp(sink)), a sink of its own per head
    q, k = torch.zeros(4, 2, 2, dtype=D), torch.zeros(4, 1, 2, dtype=D)
    v = torch.arange(4, dtype=D).reshape(4, 1, 1) + 1.0
    out = plain.attend(q, k, v, 1.0, 2, torch.tensor([0.0, math.log(3.0)], dtype=D))
    assert torch.allclose(out[:, 0, 0], torch.tensor([0.5, 1.0, 5.0 / 3, 7.0 / 3], dtype=D))
    assert torch.allclose(out[:, 1, 0], torch.tensor([0.25, 3 / 5, 1.0, 7.0 / 5], dtype=D))
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 7.0]]], dtype=D)
    f = plain.frequencies(4, 100.0, 2.0)
    assert f == [0.5, 100.0 ** -0.5 / 2.0]
    y = plain.rotate_pairs(x, [3], f, 4)
    a, b = 1.5, 3 * f[1]
    assert torch.allclose(y[0, 0], torch.tensor(
        [1 * math.cos(a) - 2 * math.sin(a), 2 * math.cos(a) + 1 * math.sin(a),
         3 * math.cos(b) - 4 * math.sin(b), 4 * math.cos(b) + 3 * math.sin(b), 7.0], dtype=D))
    u = torch.tensor([[1.0], [2.0], [3.0], [4.0]], dtype=D)
    assert plain.causal_conv(u, torch.tensor([[100.0, 10.0, 1.0]], dtype=D))[:, 0].tolist() == \
        [1.0, 12.0, 123.0, 234.0]


def test_plain_choice_of_experts_by_hand():
    s = torch.tensor([0.9, 0.1, 0.6, 0.5, 0.2, 0.3], dtype=D)
    none = torch.zeros(6, dtype=D)
    # pairs: 1.0, 1.1, 0.5: the group with the largest single score is not the best
    assert plain.group_values(s, 3) == pytest.approx([1.0, 1.1, 0.5])
    idx, w = plain.choose(s, none, 1, 3, 1, 2.0)
    assert idx == [2] and torch.allclose(w, torch.tensor([2.0], dtype=D))
    idx, w = plain.choose(s, none, 2, 3, 2, 1.0)
    assert idx == [0, 2] and torch.allclose(w, torch.tensor([0.9, 0.6], dtype=D) / 1.5)
    # the correction moves the choice, not the weights, also where all choice scores are negative
    corr = torch.tensor([-9.0, -9.0, -5.0, -5.0, -4.0, -7.0], dtype=D)
    idx, w = plain.choose(s, corr, 2, 3, 1, 1.0)
    assert idx == [2, 3] and torch.allclose(w, torch.tensor([0.6, 0.5], dtype=D) / 1.1)
    assert plain.group_values(s, 6) == pytest.approx(s.tolist())      # groups of one


def test_plain_activations():
    z = torch.tensor([-1.5, 0.5], dtype=D)
    assert torch.allclose(plain.gelu_erf(z), torch.tensor(
        [0.5 * v * (1 + math.erf(v / math.sqrt(2))) for v in (-1.5, 0.5)], dtype=D))
    assert plain.relu_squared(z).tolist() == [0.0, 0.25]


# -- caches -------------------------------------------------------------------------------
def test_readers_share_pages_and_keep_state_of_their_own():
    from inferx_b200.engine.runtime import Runtime, load_model
    from inferx_b200.weights.loader import RandomSource
    _, model = load_model(config_json=bk.BA, source=RandomSource(1), device="cpu",
                          dtype="float32", ops=host_ops)
    needs = model.cache_needs()
    # layer 1's pages are kept for its widest reader's window, layer 3 keeps every token
    assert [(g.window, g.layers) for g in groups_for(needs)] == [(0, (3,)), (9, (1,))]
    rt = Runtime(model, page_size=4, num_pages=8, max_slots=2)
    caches = rt.executor.caches
    for reader in (2, 4):
        assert caches[reader].k is caches[1].k and caches[reader].v is caches[1].v
        assert not caches[reader].writes and caches[1].writes
    assert caches[1].state["attention_conv_inputs"].shape == (2, 4, 5 * 6 + 6 + 10)
    assert caches[2].state == {} and caches[4].state == {}      # one tap, no taps: nothing kept
    assert caches[0].state["memory"].shape == (2, 3, 10, 6)
    assert caches[0].state["memory_maximum"].shape == (2, 3)
    _, model = load_model(config_json=bk.BB, source=RandomSource(1), device="cpu",
                          dtype="float32", ops=host_ops)
    caches = Runtime(model, page_size=4, num_pages=8, max_slots=2).executor.caches
    own, source = caches[2].state["attention_conv_inputs"], caches[0].state["attention_conv_inputs"]
    assert own is not source and own.shape == (2, 1, 6 * 24)
    assert source.shape == (2, 2, 6 * 24 + 2 * 24 + 2 * 40)


def test_a_layer_without_feed_forward_may_have_its_tensors_or_not(tmp_path):
    from inferx_b200.weights.safetensors_io import Checkpoint, write_safetensors
    d = bk.make_model_dir(bk.BB, tmp_path / "m", 3)
    reqs = bk.make_requests(bk.BB, [9], 3)
    ref = bk.reference_rows(d, reqs)
    path = os.path.join(d, "model.safetensors")
    ck = Checkpoint(d)
    held = {n: ck.get(n).clone() for n in ck.names()}
    ck.close()
    assert "l3.hc2.mix" in held and "l3.norm2" in held
    for keep in (True, False):
        tensors = [(n, t) for n, t in held.items()
                   if keep or not n.startswith(("l3.hc2", "l3.norm2"))]
        write_safetensors(path, iter(tensors), metadata={"format": "pt"})
        sess = ReplaySession(d, "float32", 64, page_size=4, max_live=1, device="cpu", ops=host_ops)
        mc.compare(mc.run_trace(sess, traces.whole(reqs)), ref, 2e-5, f"kept {keep}")


# -- the engine's host logic ---------------------------------------------------------
@pytest.mark.parametrize("name,cfg,seed,lengths,page", CASES)
@pytest.mark.parametrize("kind", list(mc.TRACE_KINDS))
def test_replay_matches_plain(tmp_path, name, cfg, seed, lengths, page, kind):
    d = bk.make_model_dir(cfg, tmp_path / "m", seed)
    reqs = bk.make_requests(cfg, lengths, seed)
    ref = bk.reference_rows(d, reqs)
    steps = mc.TRACE_KINDS[kind](reqs)
    sess = ReplaySession(d, "float32", traces.peak_tokens(steps), page_size=page, max_live=4,
                         device="cpu", ops=host_ops)
    rows = mc.run_trace(sess, steps)
    mc.compare(rows, ref, 2e-5, f"{name}/{kind}")
    if kind in ("whole", "tail", "portions"):
        assert len(rows) == sum(lengths)


def test_portions_of_two_tokens_and_single_tokens_agree_with_whole(tmp_path):
    d = bk.make_model_dir(bk.BA, tmp_path / "m", 7)
    toks = bk.make_requests(bk.BA, [27], 3)["r0"]
    ref = bk.reference_rows(d, {"a": toks})
    for size in (2, 1, 3, 5):
        steps = [{"step": i, "entries": [{"id": "a", "tokens": toks[a:a + size],
                                          "want": list(range(len(toks[a:a + size])))}],
                  "end": ["a"] if a + size >= len(toks) else []}
                 for i, a in enumerate(range(0, len(toks), size))]
        sess = ReplaySession(d, "float32", 64, page_size=4, max_live=1, device="cpu",
                             ops=host_ops)
        rows = mc.run_trace(sess, steps)
        assert len(rows) == len(toks)
        mc.compare(rows, ref, 2e-5, f"portions of {size}")


def test_state_slot_of_a_finished_request_starts_anew(tmp_path):
    """Two requests one after the other in a pool with one slot: the second must see neither
    the first one's memory and its maximum nor the inputs its convolutions kept."""
    for cfg in (bk.BA, bk.BD):
        d = bk.make_model_dir(cfg, tmp_path / str(cfg["width"]), 2)
        reqs = bk.make_requests(cfg, [12, 9], 5)
        ref = bk.reference_rows(d, reqs)
        sess = ReplaySession(d, "float32", 64, page_size=4, max_live=1, device="cpu", ops=host_ops)
        rows = mc.run_trace(sess, traces.whole(reqs))
        mc.compare(rows, ref, 2e-5, "slot reuse")


def test_another_norm_on_several_streams():
    """A norm that needs the whole row reads the streams through the same block: the reading
    is formed first, then normed."""
    from inferx_b200.parts.base import BuildContext, StreamUpdate
    from inferx_b200.parts.norm import RmsNorm
    from inferx_b200.parts.specs import RmsNormSpec
    from inferx_b200.parts.streams import read_streams
    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"), ops=host_ops)
    norm = RmsNorm(RmsNormSpec(12, 1e-6, suffix=""), ctx, "n")
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g)
    norm.bind({"n": r(12)})
    x, up, read = r(5, 3, 12), StreamUpdate(r(5, 12), r(3, 3), r(3)), r(3)
    new = torch.einsum("tsw,so->tow", x, up.mix) + up.put[None, :, None] * up.y[:, None, :]
    u = (read[None, :, None] * new).sum(1)
    out = read_streams(host_ops, norm, x, up, read)
    want = u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-6) * norm.gain
    assert torch.allclose(out, want, atol=1e-5) and torch.allclose(x, new, atol=1e-6)


def test_the_elementwise_norm_on_a_plain_stream():
    from inferx_b200.parts.base import BuildContext, PendingSum
    from inferx_b200.parts.norm import DynamicTanh
    from inferx_b200.parts.specs import DynamicTanhSpec
    ctx = BuildContext(dtype=torch.float32, device=torch.device("cpu"), ops=host_ops)
    norm = DynamicTanh(DynamicTanhSpec(8), ctx, "n")
    g = torch.Generator().manual_seed(2)
    r = lambda *s: torch.randn(*s, generator=g)
    w = {"n": r(8), "n.b": r(8), "n.alpha": torch.tensor(0.4)}
    norm.bind(w)
    x, y = r(3, 8), r(3, 8)
    a = x.clone()
    out = norm.forward(a, PendingSum(terms=[y], dtype=torch.float32, scale=0.5))
    assert torch.allclose(a, x + 0.5 * y)
    assert torch.allclose(out, torch.tanh(0.4 * a) * w["n"] + w["n.b"])


def test_greedy_generation_through_the_engine(tmp_path):
    from inferx_b200 import Engine, EngineConfig, Request, SamplingParams
    for cfg in (bk.BB, bk.BD):
        d = bk.make_model_dir(cfg, tmp_path / str(cfg["width"]), 4)
        c, w = plain.read_model_folder(d)
        prompts = list(bk.make_requests(cfg, [7, 19, 3], 8).values())
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
    d = bk.make_model_dir(bk.BA, tmp_path / "m", 0)
    reqs = bk.make_requests(bk.BA, [5, 9, 17], 0)

    def run(pages):
        eng = Engine.create(EngineConfig(model=d, dtype="float32", device="cpu", block_size=4,
                                         max_num_seqs=3, num_gpu_blocks_override=pages,
                                         max_model_len=64), ops=host_ops)
        outs = eng.generate([Request(t, SamplingParams(max_tokens=8, ignore_eos=True))
                             for t in reqs.values()])
        return [c.output_tokens for c in outs], eng.stats()["preemptions"]
    roomy, p0 = run(64)
    tight, p1 = run(10)
    assert p0 == 0 and p1 >= 1 and roomy == tight

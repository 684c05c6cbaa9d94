"""The Biguzen design on the GPU: every new kernel and kernel option alone against its plain
statement (tests/host_ops.py), then the engine against the plain model
(tests/plain_biguzen.py): whole prompts, prefill against token-by-token decoding, portions
down to two tokens, unequal batches with pages and slots used again, long decoding with
recorded steps over windows, and greedy generation through the engine's own entry point."""
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import biguzen_cases as bk
import host_ops
import model_cases as mc
import plain_biguzen as plain
import traces
from conftest import ROOT
from inferx_b200.engine.replay import ReplaySession
from inferx_b200.parts.base import StreamUpdate

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
CASES = [("BA", bk.BA, 0, [5, 9, 17, 40, 3, 70], 4), ("BB", bk.BB, 1, [1, 6, 13, 31, 45, 80], 8),
         ("BC", bk.BC, 2, [130, 2, 64, 33], 16), ("BD", bk.BD, 3, [70, 1, 12, 90], 16)]


def _ops():
    from inferx_b200.kernels import ops
    return ops


def _tol(dtype):
    return dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1.6e-2, atol=1.6e-2)


def _step(q_lens, starts, slots=None):
    """A batch description: sequence s brings q_lens[s] tokens from position starts[s];
    single tokens come first."""
    assert list(q_lens) == sorted(q_lens, key=lambda n: n != 1), "single tokens come first"
    seq_of, pos, cu = [], [], [0]
    for s, (n, a) in enumerate(zip(q_lens, starts)):
        seq_of += [s] * n
        pos += list(range(a, a + n))
        cu.append(cu[-1] + n)
    nd = sum(1 for n in q_lens if n == 1)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32)
    return SimpleNamespace(
        seq_of_token=i32(seq_of), positions=i32(pos), cu_q=i32(cu), q_pos0=i32(list(starts)),
        q_lens=list(q_lens), num_seqs=len(q_lens), num_tokens=len(seq_of),
        kv_len=i32([a + n for n, a in zip(q_lens, starts)]),
        max_kv_len=max(a + n for n, a in zip(q_lens, starts)), max_q_len=max(q_lens),
        all_decode=nd == len(q_lens), num_decode_seqs=nd,
        cu_q_prompt=i32([c - nd for c in cu[nd:]]),
        state_slot=i32(slots if slots is not None else list(range(len(q_lens)))))


def _cuda(x):
    if torch.is_tensor(x):
        return x.cuda()
    return SimpleNamespace(**{k: (v.cuda() if torch.is_tensor(v) else v)
                              for k, v in vars(x).items()})


def _rand(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *shape: torch.randn(*shape, generator=g)


# -- streams and the elementwise norm -----------------------------------------------------
def _update(r, y, n):
    return StreamUpdate(y, r(n, n), r(n))


def _gpu_update(u):
    return StreamUpdate(u.y.cuda() if torch.is_tensor(u.y) else u.y, u.mix.cuda(), u.put.cuda())


@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 8, 11])
@pytest.mark.parametrize("W", [60, 97, 512])
@pytest.mark.parametrize("out_dtype", DTYPES)
def test_stream_step(n, W, out_dtype):
    r = _rand(n * W)
    T = 9
    for y_dtype in DTYPES:
        x, y = r(T, n, W), r(T, W).to(y_dtype)
        up, read = _update(r, y, n), r(n)
        norm = (torch.tensor([0.7]), r(W), r(W))
        rows = torch.tensor([7, 0, 3, 3], dtype=torch.int32)
        for update in (None, up):
            for nm in (norm, None):
                for pick in (None, rows):
                    a, b = x.clone(), x.clone().cuda()
                    ref = host_ops.stream_step(a, update, read, nm, out_dtype, rows=pick)
                    got = _ops().stream_step(
                        b, None if update is None else _gpu_update(update), read.cuda(),
                        None if nm is None else tuple(t.cuda() for t in nm), out_dtype,
                        rows=None if pick is None else pick.cuda())
                    assert got.dtype == (torch.float32 if nm is None else out_dtype)
                    torch.testing.assert_close(got.cpu().float(), ref.float(), **_tol(got.dtype))
                    torch.testing.assert_close(b.cpu(), a, rtol=2e-5, atol=2e-5)
                    if update is None or pick is not None:
                        assert torch.equal(b.cpu(), x)       # nothing was written


def test_stream_update_reads_the_old_streams_and_its_matrix_is_from_to():
    """One stream holds ones; the matrix sends it to exactly one other."""
    n, W = 4, 64
    x = torch.zeros(1, n, W)
    x[0, 2] = 1.0
    mix = torch.zeros(n, n)
    mix[2, 1] = 5.0                      # from 2 to 1
    put = torch.tensor([0.0, 0.0, 0.0, 3.0])
    y = torch.full((1, W), 2.0)
    b = x.clone().cuda()
    u = _ops().stream_step(b, StreamUpdate(y.cuda(), mix.cuda(), put.cuda()),
                           torch.tensor([1.0, 10.0, 100.0, 1000.0]).cuda(), None, torch.float32)
    assert b[0, :, 0].tolist() == [0.0, 5.0, 0.0, 6.0] and float(u[0, 0]) == 6050.0


@pytest.mark.parametrize("shared", [False, True])
def test_stream_step_combines_a_mixtures_rows(shared):
    ops, r = _ops(), _rand(5)
    T, W, k, n = 13, 64, 3, 4
    y = r(T * k, W).to(torch.bfloat16)
    dest = torch.randperm(T * k).to(torch.int32)
    w = torch.rand(T, k)
    sh = r(T, W).to(torch.bfloat16) if shared else None
    logit = r(T) if shared else None
    d = sum(w[:, j, None] * y[dest.view(T, k)[:, j].long()].float() for j in range(k))
    if shared:
        d = d + torch.sigmoid(logit)[:, None] * sh.float()
    up, read, norm = _update(r, d, n), r(n), (torch.tensor([0.5]), r(W), r(W))
    x = r(T, n, W)
    a, b = x.clone(), x.clone().cuda()
    ref = host_ops.stream_step(a, up, read, norm, torch.bfloat16)
    pend = ops.CombinePending(y.cuda(), dest.cuda(), w.cuda(), sh.cuda() if shared else None,
                              logit.cuda() if shared else None)
    got = ops.stream_step(b, StreamUpdate(pend, up.mix.cuda(), up.put.cuda()), read.cuda(),
                          tuple(t.cuda() for t in norm), torch.bfloat16)
    torch.testing.assert_close(b.cpu(), a, rtol=2e-5, atol=2e-5)
    torch.testing.assert_close(got.cpu().float(), ref.float(), **_tol(torch.bfloat16))


def test_embedding_in_every_stream():
    table = _rand(1)(31, 52).to(torch.bfloat16)
    ids = torch.tensor([30, 0, 7, 7], dtype=torch.int32)
    out = _ops().embed_streams(table.cuda(), ids.cuda(), 3).cpu()
    assert torch.equal(out, host_ops.embed_streams(table, ids, 3))


# -- the matrix memory ----------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,W,cap,q_lens", [(3, 60, 4.0, [1, 1, 5, 300]), (2, 96, 15.0, [700]),
                                            (4, 64, 30.0, [1, 1, 1]), (1, 37, 2.0, [1, 2, 256, 257])])
def test_memory_gates(dtype, H, W, cap, q_lens):
    r = _rand(H * W)
    step = _step(q_lens, [3] * len(q_lens), slots=list(range(len(q_lens)))[::-1])
    T = step.num_tokens
    x, w, b = r(T, W).to(dtype), (r(2 * H, W) * 0.3).to(dtype), r(2 * H) * 3.0
    m = r(len(q_lens) + 1, H) * 2.0
    ref_m, got_m = m.clone(), m.clone().cuda()
    ref = host_ops.memory_gates(x, w, b, cap, ref_m, step)
    got = _ops().memory_gates(x.cuda(), w.cuda(), b.cuda(), cap, got_m, _cuda(step)).cpu()
    torch.testing.assert_close(got, ref, rtol=3e-4, atol=3e-5)
    torch.testing.assert_close(got_m.cpu(), ref_m, rtol=1e-4, atol=1e-4)
    assert torch.equal(got_m[-1].cpu(), m[-1])          # a slot nobody uses


def _memory_case(seed, H, K, V, q_lens, dtype, forget=2.0):
    r = _rand(seed)
    step = _step(q_lens, [2] * len(q_lens), slots=list(range(len(q_lens)))[::-1])
    T = step.num_tokens
    rows = r(T, 2 * H * K + H * V + 5).to(dtype)
    z = r(T, 2 * H)
    i, f = z[:, :H] * 2.0, torch.nn.functional.logsigmoid(z[:, H:] * 2.0 + forget)
    gates = torch.zeros(4, H, T)
    for s in range(step.num_seqs):
        m = torch.zeros(H)
        for t in range(int(step.cu_q[s]), int(step.cu_q[s + 1])):
            new = torch.maximum(f[t] + m, i[t])
            gates[0, :, t], gates[1, :, t] = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
            gates[2, :, t], gates[3, :, t] = torch.exp(-new), f[t] + m - new
            m = new
    S, n = r(len(q_lens) + 1, H, K, V), r(len(q_lens) + 1, H, K)
    return step, rows, gates, S, n


def _views(rows, H, K, V):
    return rows[:, :H * K], rows[:, H * K:2 * H * K], rows[:, 2 * H * K:2 * H * K + H * V]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,K,V", [(3, 10, 6), (3, 40, 48), (2, 64, 128), (1, 130, 36), (1, 24, 200),
                                   (2, 16, 7)])
@pytest.mark.parametrize("q_lens", [[1, 1, 1], [1, 5, 2], [1, 1, 200, 64, 65], [31], [321]])
def test_matrix_memory(dtype, H, K, V, q_lens):
    step, rows, gates, S, n = _memory_case(K + V, H, K, V, q_lens, dtype)
    refS, refn = S.clone(), n.clone()
    num, nq = host_ops.matrix_memory(*_views(rows, H, K, V), gates, refS, refn, step, H, K, V, 0.3)
    forms = ["walk"] + (["chunks"] if dtype == torch.bfloat16 and max(q_lens) > 1 else [])
    for form in forms:
        gS, gn = S.clone().cuda(), n.clone().cuda()
        a, b = _ops().matrix_memory(*_views(rows.cuda(), H, K, V), gates.cuda(), gS, gn,
                                    _cuda(step), H, K, V, 0.3, form=form)
        rel = 2e-5 if form == "walk" else 6e-5      # start states and weights of 16 bits
        for got, ref in ((a, num), (b, nq), (gS, refS), (gn, refn)):
            err = float((got.cpu() - ref).abs().max()) / float(ref.abs().max())
            assert err < rel, (form, err)
        assert torch.equal(gS[-1].cpu(), S[-1]) and torch.equal(gn[-1].cpu(), n[-1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,K,V", [(3, 10, 6), (3, 40, 48), (2, 64, 128), (1, 24, 200), (2, 16, 7)])
@pytest.mark.parametrize("q_lens", [[1, 1, 1], [1, 5, 2], [1, 1, 200, 64, 65], [100]])
def test_matrix_memory_finishes_the_heads(dtype, H, K, V, q_lens):
    """Division by the normaliser, norm, gain and gate in the memory's kernels where a block has
    the whole head, else behind them."""
    step, rows, gates, S, n = _memory_case(K + V + 1, H, K, V, q_lens, dtype)
    r = _rand(V)
    T = step.num_tokens
    gain, gate = r(H * V), r(T, H * V + 2 * (V % 2) + 4).to(dtype)
    n = n * 0.02                                     # some denominators are the floor's
    refS, refn = S.clone(), n.clone()
    ref = host_ops.matrix_memory(*_views(rows, H, K, V), gates, refS, refn, step, H, K, V, 0.3,
                                 finish=(gain, gate[:, :H * V], 1e-5, 1e-6)).float()
    for form in ["walk"] + (["chunks"] if dtype == torch.bfloat16 and max(q_lens) > 1 else []):
        gS, gn = S.clone().cuda(), n.clone().cuda()
        y = _ops().matrix_memory(*_views(rows.cuda(), H, K, V), gates.cuda(), gS, gn, _cuda(step),
                                 H, K, V, 0.3, form=form,
                                 finish=(gain.cuda(), gate.cuda()[:, :H * V], 1e-5, 1e-6))
        assert y.dtype == dtype
        err = (y.cpu().float() - ref).abs().max() / ref.abs().max()
        assert float(err) < (3e-4 if dtype == torch.float32 else 1e-2), (form, float(err))
        assert float((gS.cpu() - refS).abs().max() / refS.abs().max()) < 6e-5


@pytest.mark.parametrize("form,dtype", [("walk", torch.float32), ("walk", torch.bfloat16),
                                        ("chunks", torch.bfloat16)])
def test_memory_carries_what_was_written_far_back(form, dtype):
    """One token writes a strong pair, the next 400 write nothing and forget nothing; the last
    query asks with the same key and finds the value.  The portions end at the borders of
    chunks and beside them."""
    H, K, V = 1, 32, 48
    for cuts in ([401], [64, 337], [63, 2, 65, 271], [1, 400], [17] * 23 + [10]):
        S, n = torch.zeros(1, H, K, V).cuda(), torch.zeros(1, H, K).cuda()
        rows = torch.zeros(401, 2 * K + V)
        rows[0, K:2 * K], rows[0, 2 * K:] = 1.0, 3.0       # key of ones, value of threes
        rows[400, :K] = 1.0                                # the query
        gates = torch.zeros(4, H, 401)
        gates[0], gates[1], gates[2], gates[3] = 1.0, 0.0, 1.0, 0.0
        gates[1, :, 0] = 0.5
        at, last = 0, None
        for c in cuts:
            step = _cuda(_step([c], [at]))
            part = rows[at:at + c].to(dtype).cuda()
            f = None if c == 1 else form
            num, nq = _ops().matrix_memory(*_views(part, H, K, V),
                                           gates[:, :, at:at + c].contiguous().cuda(), S, n, step, H,
                                           K, V, 1.0, form=f)
            at, last = at + c, (num[-1], nq[-1])
        assert at == 401
        assert torch.allclose(last[0].cpu(), torch.full((H, V), 0.5 * K * 3.0))
        assert torch.allclose(last[1].cpu(), torch.full((H,), 0.5 * K))


def test_memory_does_not_depend_on_the_cut_or_the_batch():
    """A sequence whole, in portions, and in portions beside other sequences."""
    H, K, V, T = 2, 48, 80, 230
    step, rows, gates, S, n = _memory_case(4, H, K, V, [T], torch.bfloat16)
    gS, gn = S.clone().cuda(), n.clone().cuda()
    whole, wq = _ops().matrix_memory(*_views(rows.cuda(), H, K, V), gates.cuda(), gS, gn,
                                     _cuda(step), H, K, V, 0.2)
    other = _memory_case(5, H, K, V, [1, 90], torch.bfloat16)
    pS, pn = torch.cat([S, S, S]).cuda(), torch.cat([n, n, n]).cuda()
    at, nums, nqs = 0, [], []
    for c in (33, 2, 64, 100, 31):
        rs = torch.cat([other[1][:1], other[1][1:91], rows[at:at + c]])
        gs = torch.cat([other[2][:, :, :91], gates[:, :, at:at + c]], dim=2).contiguous()
        st = _cuda(_step([1, 90, c], [0, 0, at], slots=[3, 4, 0]))
        a, b = _ops().matrix_memory(*_views(rs.cuda(), H, K, V), gs.cuda(), pS, pn, st, H, K, V, 0.2)
        nums.append(a[91:])
        nqs.append(b[91:])
        at += c
    for got, ref in ((torch.cat(nums), whole), (torch.cat(nqs), wq), (pS[0], gS[0]), (pn[0], gn[0])):
        assert float((got - ref).abs().max()) / float(ref.abs().max()) < 6e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("V", [6, 48, 64, 128])
@pytest.mark.parametrize("form", ["sigmoid", "silu"])
def test_head_norm_with_denominator(dtype, V, form):
    T, H, r = 11, 3, _rand(V)
    o, gain, gate = r(T, H, V), r(H * V), r(T, H * V + 3).to(dtype)
    nq, floor = r(T, H), torch.rand(H, T)
    nq[0], floor[:, 0] = 0.0, 0.0                  # the added constant alone divides
    for den in (None, (nq, floor, 1e-6)):
        ref = host_ops.head_norm_gate(o, gain, gate[:, :H * V], 1e-5, dtype, form, den=den)
        got = _ops().head_norm_gate(o.cuda(), gain.cuda(), gate.cuda()[:, :H * V], 1e-5, dtype, form,
                                    den=None if den is None else (nq.cuda(), floor.cuda(), 1e-6))
        torch.testing.assert_close(got.cpu().float(), ref.float(), **_tol(dtype))


# -- attention's options ----------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps", [(40, 1), (64, 3), (37, 5), (128, 4)])
@pytest.mark.parametrize("q_lens", [[1, 1, 7], [2, 1100], [3], [1, 1, 1, 1]])
def test_convolution_adds_its_input_bias_first(dtype, C, taps, q_lens):
    q_lens = sorted(q_lens, key=lambda n: n != 1)
    r = _rand(C + taps)
    step = _step(q_lens, [0] * len(q_lens))
    x, w, b = r(step.num_tokens, C + 8).to(dtype), r(C, taps), r(C)
    state = r(len(q_lens), max(1, taps - 1), C)
    ref_s, got_s = state.clone(), state.clone().cuda()
    args = (None if taps == 1 else ref_s,), (None if taps == 1 else got_s,)
    ref = host_ops.causal_conv(x[:, :C], w, None, *args[0], step, silu=False, in_bias=b)
    got = _ops().causal_conv(x.cuda()[:, :C], w.cuda(), None, *args[1], _cuda(step), silu=False,
                             in_bias=b.cuda())
    torch.testing.assert_close(got.cpu().float(), ref.float(), **_tol(dtype))
    torch.testing.assert_close(got_s.cpu(), ref_s, rtol=1e-6, atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,rot", [(5, 6, 4), (6, 24, 12), (4, 128, 32), (3, 64, 0)])
def test_preparation_of_queries_alone(dtype, H, D, rot):
    r = _rand(H * D)
    T = 19
    row = r(T, H * D + 8).to(dtype)
    pos = torch.arange(1000, 1000 + T, dtype=torch.int32)
    freq = torch.rand(rot // 2) if rot else None
    args = (1.0, rot, True, H, 0, D, D, None, None, 1e-6, False, None, None, None, None, None)
    ref = host_ops.attention_prepare(row[:, :H * D], pos, freq, *args)
    got = _ops().attention_prepare(row.cuda()[:, :H * D], pos.cuda(),
                                   None if freq is None else freq.cuda(), *args)
    torch.testing.assert_close(got.cpu().float(), ref.float(), rtol=1.6e-2, atol=2e-3)


def _kv_case(seed, H, G, D, VD, page, q_lens, starts, dtype):
    g = torch.Generator().manual_seed(seed)
    step = _step(q_lens, starts)
    need = [-(-(a + n) // page) for n, a in zip(q_lens, starts)]
    total = sum(need) + 3
    perm = torch.randperm(total, generator=g).to(torch.int32)
    bt = torch.full((len(q_lens), max(need)), -1, dtype=torch.int32)
    at = 0
    for s, n in enumerate(need):
        bt[s, :n] = perm[at:at + n]
        at += n
    kc = (torch.randn(total, G, page, D, generator=g) * 0.5).to(dtype)
    vc = torch.randn(total, G, page, VD, generator=g).to(dtype)
    q = torch.randn(step.num_tokens, H, D, generator=g).to(dtype)
    sink = torch.randn(H, generator=g) * 2.0
    gate = torch.randn(step.num_tokens, H + 3, generator=g).to(dtype)
    return step, bt, kc, vc, q, sink, gate


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,VD", [(5, 1, 6, 10), (6, 2, 24, 40), (8, 2, 64, 64), (4, 4, 64, 128),
                                      (16, 1, 128, 128), (5, 1, 128, 64)])
@pytest.mark.parametrize("window", [0, 1, 40])
@pytest.mark.parametrize("q_lens,starts", [([1, 1, 1], [0, 39, 700]), ([150, 2], [0, 77]),
                                           ([1, 1, 70], [200, 5, 30])])
def test_attention_with_learned_sinks_and_head_gates(dtype, H, G, D, VD, window, q_lens, starts):
    page, scale = 16, 1.3 * D ** -0.5
    step, bt, kc, vc, q, sink, gate = _kv_case(H + D + window, H, G, D, VD, page, q_lens, starts,
                                               dtype)
    ops, cs = _ops(), _cuda(step)
    dev = [t.cuda() for t in (q, kc, vc, bt)]
    for sk, gt in ((sink, gate[:, :H]), (sink, None), (None, gate[:, :H])):
        ref = host_ops.paged_attention(q, kc, vc, bt, step, window, scale, sink=sk, gate=gt).float()
        opt = dict(sink=None if sk is None else sk.cuda(),
                   gate=None if gt is None else gate.cuda()[:, :H])
        got = ops.paged_attention(*dev, cs, window, scale, fp32_weights=True, **opt)
        torch.testing.assert_close(got.cpu().float(), ref, **_tol(dtype))
        gen = ops.paged_attention_generic(*dev, cs.seq_of_token, cs.positions, window, scale, **opt)
        torch.testing.assert_close(gen.cpu().float(), ref, **_tol(dtype))
        if D % 4 == 0 and VD % 4 == 0:
            til = ops.paged_attention_tiled(*dev, cs.cu_q, cs.q_pos0, window, scale, **opt)
            torch.testing.assert_close(til.cpu().float(), ref, **_tol(dtype))
        if step.all_decode:
            for splits in (None, 1, 7):
                got = ops.paged_attention_decode_any(*dev, cs.kv_len, cs.max_kv_len, window, scale,
                                                     splits=splits, **opt)
                torch.testing.assert_close(got.cpu().float(), ref, **_tol(dtype))
        if dtype == torch.bfloat16 and D in (64, 128):
            if step.all_decode:
                for splits in (1, 5):
                    got = ops.paged_attention_decode_exact(*dev, cs.kv_len, cs.max_kv_len, window,
                                                           scale, splits=splits, **opt)
                    torch.testing.assert_close(got.cpu().float(), ref, **_tol(dtype))
            for kernel in ("mma",) + (("tc",) if D == VD else ()):
                got = ops.paged_attention_prefill_exact(*dev, cs.cu_q, cs.q_pos0, window, scale,
                                                        kernel=kernel, **opt)
                torch.testing.assert_close(got.cpu().float(), ref, **_tol(dtype))
    ops.check_async_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,VD", [(24, 40), (64, 64), (128, 128)])
@pytest.mark.parametrize("decode", [True, False])
def test_a_window_s_last_key_is_seen_and_the_key_before_it_is_not(dtype, D, VD, decode):
    """One key carries a score far above the rest (and above the sink) and a value of fives."""
    window, query_pos, page, H, scale = 40, 700, 16, 2, D ** -0.5
    for key_pos, seen in ((700, True), (661, True), (660, False), (672, True), (0, False)):
        n0 = 1 if decode else 9
        step, bt, kc, vc, q, sink, _ = _kv_case(key_pos, H, 1, D, VD, page, [n0],
                                                [query_pos - n0 + 1], dtype)
        qv = q[n0 - 1, 0].float()
        q[n0 - 1, 1] = q[n0 - 1, 0]
        pg, off = int(bt[0, key_pos // page]), key_pos % page
        kc[pg, 0, off] = (qv * (60.0 / scale) / (qv * qv).sum()).to(dtype)
        vc[pg, 0, off] = 5.0
        out = _ops().paged_attention(q.cuda(), kc.cuda(), vc.cuda(), bt.cuda(), _cuda(step), window,
                                     scale, fp32_weights=True, sink=sink.cuda()).cpu().float()
        assert (float(out[n0 - 1].mean()) > 4.9) == seen, key_pos


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("decode", [True, False])
@pytest.mark.parametrize("D", [24, 64])
def test_each_head_has_a_sink_of_its_own(dtype, decode, D):
    """Scores of zero: with a sink s the weight of each of n keys is 1 / (n + exp(s)); a sink far
    above every score takes everything, one far below nothing."""
    H, page, n0 = 4, 16, 1 if decode else 30
    step, bt, kc, vc, q, _, _ = _kv_case(3, H, 2, D, D, page, [n0], [200 - n0 + 1], dtype)
    q.zero_()
    vc.fill_(1.0)
    sink = torch.tensor([-100.0, 0.0, math.log(50.0), 90.0])
    out = _ops().paged_attention(q.cuda(), kc.cuda(), vc.cuda(), bt.cuda(), _cuda(step), 50, 1.0,
                                 fp32_weights=True, sink=sink.cuda()).cpu().float()[n0 - 1]
    for h, want in enumerate((1.0, 50.0 / 51.0, 0.5, 0.0)):
        assert abs(float(out[h].mean()) - want) < 5e-3, (h, float(out[h].mean()))


# -- experts --------------------------------------------------------------------------------
@pytest.mark.parametrize("T", [3, 40, 300])
@pytest.mark.parametrize("E,k,groups,keep", [(15, 4, 3, 2), (8, 2, 8, 5), (40, 4, 4, 1), (6, 6, 2, 2)])
def test_groups_valued_by_their_two_best(T, E, k, groups, keep):
    r = _rand(T + E)
    x, w, corr = r(T, 64), r(E, 64) * 0.2, r(E) - 3.0         # every choice score is negative
    rule = dict(correction=corr, group_count=groups, group_keep=keep, renorm_eps=1e-20,
                score="sigmoid", group_value="pair_sum")
    rw, ri, _ = host_ops.router_topk(x, w, k, True, 1.7, **rule)
    rule["correction"] = corr.cuda()
    gw, gi, _ = _ops().router_topk(x.cuda(), w.cuda(), k, True, 1.7, **rule)
    same = (gi.cpu() == ri).all(-1)
    assert float(same.float().mean()) > 0.99                  # (a tie in fp32 may fall elsewhere)
    torch.testing.assert_close(gw.cpu()[same], rw[same], rtol=1e-5, atol=1e-6)
    assert torch.allclose(gw.sum(-1).cpu(), torch.full((T,), 1.7), rtol=1e-5)
    if T == 300 and groups < E and keep < groups:
        # the rule matters: the largest score alone chooses otherwise
        _, other, _ = host_ops.router_topk(x, w, k, True, 1.7, **dict(
            rule, correction=corr, group_value="max"))
        assert (other != ri).any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("activation", ["gelu", "relu_squared"])
@pytest.mark.parametrize("M,N,K", [(1, 96, 64), (7, 130, 256), (16, 33, 60), (50, 384, 256), (3, 18, 37)])
def test_dense_product_with_activation(dtype, activation, M, N, K):
    r = _rand(M + N)
    x, w = r(M, K).to(dtype), (r(N, K) * K ** -0.5 * 2).to(dtype)
    ref = host_ops.linear_act(x, w, activation)
    got = _ops().linear_act(x.cuda(), w.cuda(), activation)
    torch.testing.assert_close(got.cpu().float(), ref.float(), **_tol(dtype))
    y = r(M, N).to(dtype)
    got = _ops().activate(y.cuda(), activation)
    torch.testing.assert_close(got.cpu().float(), host_ops.activate(y, activation).float(),
                               **_tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("activation", ["gelu", "relu_squared"])
@pytest.mark.parametrize("T,E,k,H,I", [(1, 8, 2, 256, 96), (3, 4, 1, 256, 40), (9, 6, 2, 64, 48),
                                       (60, 6, 2, 60, 18), (300, 4, 2, 128, 136), (500, 3, 3, 128, 384)])
def test_experts_without_a_gate(dtype, activation, T, E, k, H, I):
    r = _rand(T + I)
    x, w = r(T, H).to(dtype), (r(E, I, H) * H ** -0.5 * 2).to(dtype)
    idx = torch.stack([torch.randperm(E)[:k] for _ in range(T)]).to(torch.int32)
    offsets, rows, _ = host_ops.moe_dispatch(idx, E)
    ref = host_ops.grouped_up(x, rows, offsets, w, activation)
    got = _ops().grouped_up(x.cuda(), rows.cuda(), offsets.cuda(), w.cuda(), activation)
    torch.testing.assert_close(got.cpu().float(), ref.float(), **_tol(dtype))
    _ops().check_async_errors()


# -- the engine against the plain model ------------------------------------------------
def _folder_dtype(dtype):
    return "float32" if dtype == "float32" else "bfloat16"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,cfg,seed,lengths,page", CASES)
@pytest.mark.parametrize("kind", list(mc.TRACE_KINDS))
def test_replay_matches_plain(tmp_path, dtype, name, cfg, seed, lengths, page, kind):
    d = bk.make_model_dir(cfg, tmp_path / "m", seed, dtype=_folder_dtype(dtype))
    reqs = bk.make_requests(cfg, lengths, seed)
    ref = bk.reference_rows(d, reqs)
    steps = mc.TRACE_KINDS[kind](reqs)
    sess = ReplaySession(d, dtype, traces.peak_tokens(steps), page_size=page, max_live=4)
    rows = bk.rows_to_compare(dtype, d, reqs, mc.run_trace(sess, steps))
    worst = mc.compare(rows, ref, bk.bound_for(dtype, d, reqs), f"{name}/{kind}/{dtype}")
    print(f"{name}/{kind}/{dtype}: worst relative error {worst:.3e}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cfg", [bk.BA, bk.BC])
def test_long_decoding_with_recorded_steps(tmp_path, dtype, cfg):
    """250 tokens one by one after a short prompt: every window passes over decoded tokens,
    pages fall behind it and are given back, memories and the convolutions' kept inputs are
    carried through recorded steps."""
    d = bk.make_model_dir(cfg, tmp_path / "m", 3, dtype=_folder_dtype(dtype))
    reqs = bk.make_requests(cfg, [270], 3)
    ref = bk.reference_rows(d, reqs)
    steps = traces.tail_decode(reqs, 250)
    sess = ReplaySession(d, dtype, traces.peak_tokens(steps), page_size=4, use_graphs=True)
    rows = mc.run_trace(sess, steps)
    assert len(rows) == 270 and sess.executor.graph_replays >= 200
    rows = bk.rows_to_compare(dtype, d, reqs, rows, share=0.005)
    mc.compare(rows, ref, bk.bound_for(dtype, d, reqs), f"long decode {dtype}")


@pytest.mark.parametrize("dtype,kind", [("bfloat16", "whole"), ("bfloat16", "mixed"),
                                        ("bfloat16", "portions"), ("float32", "tail")])
def test_long_prompts(tmp_path, dtype, kind):
    """Prompts of several hundred tokens at tensor-core sizes: many chunks of the memory, many
    key tiles, windows of two widths over the same keys, experts all chosen."""
    cfg = bk.BC
    d = bk.make_model_dir(cfg, tmp_path / "m", 11, dtype=_folder_dtype(dtype))
    reqs = bk.make_requests(cfg, [400, 260], 11)
    ref = bk.reference_rows(d, reqs)
    steps = (traces.portions(reqs, sizes=(90, 33, 2, 64, 65, 1, 127)) if kind == "portions"
             else mc.TRACE_KINDS[kind](reqs))
    sess = ReplaySession(d, dtype, traces.peak_tokens(steps), page_size=16, max_live=4)
    rows = mc.run_trace(sess, steps)
    sess.executor.poll_errors()
    rows = bk.rows_to_compare(dtype, d, reqs, rows)
    mc.compare(rows, ref, bk.bound_for(dtype, d, reqs), f"long/{kind}/{dtype}")


def test_prefill_equals_decoding_in_32_bit(tmp_path):
    """The same sequence whole, token by token and in portions of two: the three runs
    agree with each other far inside their distance to the plain model."""
    cfg = bk.BB
    d = bk.make_model_dir(cfg, tmp_path / "m", 6)
    reqs = bk.make_requests(cfg, [75], 6)
    runs = []
    for steps in (traces.whole(reqs), traces.tail_decode(reqs, 74),
                  traces.portions(reqs, sizes=(2,))):
        sess = ReplaySession(d, "float32", 128, page_size=8, max_live=1)
        rows = mc.run_trace(sess, steps)
        runs.append(torch.stack([rows[("r0", p)] for p in range(75)]))
    scale = float(runs[0].abs().max())
    for other in runs[1:]:
        assert float((other - runs[0]).abs().max()) / scale < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_equals_each_alone(tmp_path, dtype):
    """Four requests of unequal length that advance together, prompts beside single tokens,
    against each of them alone."""
    cfg = bk.BC
    d = bk.make_model_dir(cfg, tmp_path / "m", 8, dtype=_folder_dtype(dtype))
    reqs = bk.make_requests(cfg, [90, 12, 40, 75], 8)
    alone = mc.run_trace(ReplaySession(d, dtype, 128, page_size=16, max_live=1), traces.whole(reqs))
    steps = traces.mixed(reqs, max_live=4, seed=5)
    together = mc.run_trace(ReplaySession(d, dtype, traces.peak_tokens(steps), page_size=16,
                                          max_live=4), steps)
    scale = max(float(v.abs().max()) for v in alone.values())
    worst = max(float((v - alone[k]).abs().max()) for k, v in together.items()) / scale
    assert worst < (1e-5 if dtype == "float32" else bk.bound_for(dtype, d, reqs)), worst


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(tmp_path, dtype):
    cfg = bk.BB
    d = bk.make_model_dir(cfg, tmp_path / "m", 5, dtype="bfloat16")
    reqs = bk.make_requests(cfg, [70, 33, 20, 9, 50, 41], 5)
    ref = bk.reference_rows(d, reqs)
    steps = traces.mixed(reqs, max_live=4, seed=1)
    out = tmp_path / "out"
    p = subprocess.run(
        [sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype,
         "--out", str(out), "--max-tokens", str(traces.peak_tokens(steps))],
        input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
        timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    outs = []
    for s in steps:
        n = sum(len(e["want"]) for e in s["entries"])
        outs.append(None if n == 0 else torch.from_numpy(
            np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(n, cfg["vocab"]).copy()))
    rows = bk.rows_to_compare(dtype, d, reqs, traces.collect(steps, outs))
    mc.compare(rows, ref, bk.bound_for(dtype, d, reqs), f"trace_run/{dtype}")


def _greedy_is_the_plain_models(c, w, prompt, tokens):
    seq = list(prompt)
    for tok in tokens:
        lg = plain.forward(c, w, seq)[-1]
        best = torch.topk(lg, 2).values
        # the engine's choice is the plain model's, unless the two best are a tie in fp32
        assert tok == int(lg.argmax()) or float(best[0] - best[1]) < 1e-4 * float(lg.abs().max())
        seq.append(tok)


@pytest.mark.parametrize("cfg", [bk.BA, bk.BD])
def test_greedy_generation_through_the_engine(tmp_path, cfg):
    from inferx_b200 import Engine, EngineConfig, Request, SamplingParams
    d = bk.make_model_dir(cfg, tmp_path / "m", 4)
    c, w = plain.read_model_folder(d)
    prompts = list(bk.make_requests(cfg, [7, 19, 3, 30, 11], 8).values())
    eng = Engine.create(EngineConfig(model=d, dtype="float32", block_size=4, max_num_seqs=3,
                                     num_gpu_blocks_override=96, prefill_chunk=6,
                                     max_model_len=64))
    done = eng.generate([Request(p, SamplingParams(max_tokens=12, ignore_eos=True))
                         for p in prompts])
    for p, out in zip(prompts, done):
        _greedy_is_the_plain_models(c, w, p, out.output_tokens)
        assert len(out.output_tokens) == 12


def test_command_line(tmp_path):
    d = bk.make_model_dir(bk.BB, tmp_path / "m", 9)
    c, w = plain.read_model_folder(d)
    p = subprocess.run(
        [sys.executable, os.path.join(ROOT, "bin", "inferx-generate"), d, "--dtype", "fp32",
         "--block-size", "4", "--max-model-len", "64", "--max-num-seqs", "2",
         "--num-gpu-blocks-override", "48", "--log-level", "warning", "--prompt-ids", "5,17,3,90,41",
         "--prompt-ids", "9 8 7", "--max-tokens", "6", "--ignore-eos"],
        capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    lines = [json.loads(ln) for ln in p.stdout.splitlines() if ln.startswith("{")]
    for line, prompt in zip(lines, ([5, 17, 3, 90, 41], [9, 8, 7])):
        _greedy_is_the_plain_models(c, w, prompt, line["output_ids"])
        assert len(line["output_ids"]) == 6

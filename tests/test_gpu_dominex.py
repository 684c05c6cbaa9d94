"""The Dominex design on the GPU: every new kernel and kernel option alone against its plain
statement (tests/host_ops.py), then the engine against the plain model
(tests/plain_dominex.py): whole prompts, prefill against token-by-token decoding, portions
down to two tokens, unequal batches with pages and slots used again, long decoding with
recorded steps over the borders of runs, and greedy generation through the engine's own
entry point."""
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import dominex_cases as dk
import host_ops
import model_cases as mc
import plain_dominex as plain
import traces
from conftest import ROOT
from inferx_b200.engine.replay import ReplaySession

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
CASES = [("DA", dk.DA, 0, [5, 9, 27, 44, 3, 60], 4), ("DB", dk.DB, 1, [1, 6, 13, 31, 45], 8),
         ("DC", dk.DC, 3, [21, 1, 50, 2, 110], 16)]


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
        all_decode=nd == len(q_lens), num_decode_seqs=nd, cu_q_prompt=i32([c - nd for c in cu[nd:]]),
        state_slot=i32(slots if slots is not None else list(range(len(q_lens)))))


def _cuda(ns):
    return SimpleNamespace(**{k: (v.cuda() if torch.is_tensor(v) else v)
                              for k, v in vars(ns).items()})


def _kv_case(seed, H, G, D, VD, page, q_lens, starts, dtype, chunk=0):
    """(step, block table, key pages, value pages, q rows): pages in a shuffled order, those
    that hold no key a query of this step can see given back."""
    g = torch.Generator().manual_seed(seed)
    step = _step(q_lens, starts)
    S = len(q_lens)
    need = [-(-(a + n) // page) for n, a in zip(q_lens, starts)]
    total = sum(need) + 3
    perm = torch.randperm(total, generator=g).to(torch.int32)
    bt = torch.full((S, max(need)), -1, dtype=torch.int32)
    at = 0
    for s, n in enumerate(need):
        bt[s, :n] = perm[at:at + n]
        at += n
        if chunk > 0:
            bt[s, :starts[s] // chunk * chunk // page] = -1
    kc = (torch.randn(total, G, page, D, generator=g) * 0.4).to(dtype)
    vc = torch.randn(total, G, page, VD, generator=g).to(dtype)
    q = (torch.randn(sum(q_lens), H * D, generator=g) * 0.4).to(dtype)
    return step, bt, kc, vc, q


def _head_vectors(H, seed):
    g = torch.Generator().manual_seed(seed)
    return (0.5 + torch.rand(H, generator=g), torch.rand(H, generator=g) * 1.5,
            torch.rand(H, generator=g) * 0.6)


def _wide(t, lead, tail, seed=0):
    """``t`` as a view of columns of a wider tensor on the device."""
    w = torch.randn(t.shape[0], lead + t.shape[1] + tail,
                    generator=torch.Generator().manual_seed(seed)).to(t.dtype)
    w[:, lead:lead + t.shape[1]] = t
    return w.cuda()[:, lead:lead + t.shape[1]]


# -- kernels alone -------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("G,D,VD,page,lead", [(2, 16, 24, 4, 8), (1, 7, 9, 8, 3), (3, 64, 128, 16, 0),
                                              (2, 64, 64, 16, 5)])
def test_key_and_value_rows_into_pages(dtype, G, D, VD, page, lead):
    g = torch.Generator().manual_seed(G * D)
    T, pages = 13, 6
    k, v = (torch.randn(T, G * n, generator=g).to(dtype) for n in (D, VD))
    slots = torch.randperm(pages * page, generator=g)[:T].to(torch.int32)
    kc, vc = (torch.zeros(pages, G, page, n, dtype=dtype) for n in (D, VD))
    dk_, dv_ = kc.cuda(), vc.cuda()
    host_ops.append_kv_rows(k, v, kc, vc, slots)
    _ops().append_kv_rows(_wide(k, lead, 16), _wide(v, lead, 8, 1), dk_, dv_, slots.cuda())
    assert torch.equal(dk_.cpu(), kc) and torch.equal(dv_.cpu(), vc)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,lead", [(31, 3), (56, 8), (16, 0), (384, 4), (2050, 2)])
@pytest.mark.parametrize("q_lens", [[1, 1, 1], [1, 1, 3, 40, 2], [511], [700], [1, 9, 520, 1025],
                                    [64, 4100]])
def test_gated_recurrence(dtype, W, lead, q_lens):
    """Single tokens, portions shorter and longer than a stretch of the walk, and both kinds
    in one batch; the state comes from and goes back to each sequence's slot."""
    g = torch.Generator().manual_seed(W + len(q_lens))
    T, S = sum(q_lens), len(q_lens)
    front = (torch.randn(T, 3 * W, generator=g) * 2.0).to(dtype)
    zb, xb = torch.randn(W, generator=g) - 1.5, torch.randn(W, generator=g)
    slots = torch.randperm(S + 2, generator=g)[:S].tolist()
    step = _step(q_lens, [5] * S, slots)
    state = torch.randn(S + 2, W, generator=g)
    ref_state, dev_state = state.clone(), state.cuda()
    ref = host_ops.min_gru(front, zb, xb, 0.5, ref_state, step, torch.empty(T, W), 1.3)
    wide = torch.full((T, W + 2 * lead + 2), 7.0, dtype=dtype, device="cuda")
    off = 2 * lead
    _ops().min_gru(_wide(front, off, 6), zb.cuda(), xb.cuda(), 0.5, dev_state, _cuda(step),
                   wide[:, off:off + W], 1.3)
    torch.testing.assert_close(wide[:, off:off + W].float().cpu(), ref, **_tol(dtype))
    tol = 3e-5 if dtype == torch.float32 else 1e-4
    torch.testing.assert_close(dev_state.cpu(), ref_state, rtol=tol, atol=tol)
    others = [i for i in range(S + 2) if i not in slots]
    assert torch.equal(dev_state.cpu()[others], state[others])
    assert bool((wide[:, :off] == 7).all()) and bool((wide[:, off + W:] == 7).all())


@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_recurrence_carries_what_was_written_far_back(dtype):
    """Gates that are almost shut after the first token: its candidate must survive a thousand
    tokens of a walk in pieces, and a cut anywhere gives the same state."""
    W, n = 40, 1300
    front = torch.zeros(n, 3 * W)
    front[:, :W] = -14.0
    front[0, :W] = 14.0
    front[:, W:2 * W] = -3.0
    front[0, W:2 * W] = torch.linspace(1.0, 50.0, W)
    front[:, 2 * W:] = 2.0
    front = front.to(dtype)
    zero = torch.zeros(W)
    finals = []
    for cuts in ([n], [1, n - 1], [2, 511, 514, n - 1027], [700, 600]):
        state, out, at = torch.zeros(1, W).cuda(), torch.empty(n, W, dtype=dtype, device="cuda"), 0
        for c in cuts:
            _ops().min_gru(front[at:at + c].cuda(), zero.cuda(), zero.cuda(), 0.5, state,
                           _cuda(_step([c], [at])), out[at:at + c], 1.0)
            at += c
        finals.append((state.cpu(), out.float().cpu()))
    ref_state = torch.zeros(1, W)
    ref = host_ops.min_gru(front, zero, zero, 0.5, ref_state, _step([n], [0]), torch.empty(n, W))
    assert float(ref_state.max()) > 40.0
    # 1 - z of a gate of 8e-7 is rounded to fp32 at every token: n * 2^-25 in all
    tol = dict(rtol=1e-4, atol=1e-4) if dtype == torch.float32 else _tol(dtype)
    for st, out in finals:
        torch.testing.assert_close(st, ref_state, rtol=1e-4, atol=1e-4)
        torch.testing.assert_close(out, ref, **tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,rank,dr,rot,own", [(28, 24, 8, 8, True), (9, 11, 2, 2, True),
                                                    (1536, 512, 64, 64, True), (112, 0, 0, 0, False),
                                                    (20, 16, 6, 4, True)])
def test_query_latent_and_record(dtype, q_rank, rank, dr, rot, own):
    g = torch.Generator().manual_seed(q_rank)
    T, page, pages = 7, 4, 5
    proj = (torch.randn(T, q_rank + rank + dr + 3, generator=g) * 2.0).to(dtype)
    qg = 1.0 + 0.3 * torch.randn(q_rank, generator=g)
    kg = 1.0 + 0.3 * torch.randn(max(rank, 1), generator=g)
    pos = torch.tensor([0, 1, 2, 900, 901, 65, 7], dtype=torch.int32)
    freq = torch.rand(rot // 2, generator=g)
    slots = torch.randperm(page * pages, generator=g)[:T].to(torch.int32)
    cache = torch.zeros(pages, 1, page, rank + dr, dtype=dtype) if own else None
    dev = cache.cuda() if own else None
    args = (q_rank, qg, 1e-5, q_rank, pos, freq, 1.0, kg if own else None, rank, dr, rot)
    ref = host_ops.latent_front(proj, *args, cache, slots if own else None)
    out = _ops().latent_front(proj.cuda(), *[a.cuda() if torch.is_tensor(a) else a for a in args],
                              dev, slots.cuda() if own else None)
    torch.testing.assert_close(out.cpu().float(), ref.float(), **_tol(dtype))
    if own:
        torch.testing.assert_close(dev.cpu().float(), cache.float(), **_tol(dtype))
    # the queries a latent is widened to, split and turned
    H, dim = 3, 5
    rd = max(rot, 2)
    q = torch.randn(T, H * (dim + rd), generator=g).to(dtype)
    f2 = torch.rand(rd // 2, generator=g)
    want = host_ops.latent_queries(q, pos, f2, 1.0, H, dim, rd, rd)
    got = _ops().latent_queries(q.cuda(), pos.cuda(), f2.cuda(), 1.0, H, dim, rd, rd)
    for a, b in zip(got, want):
        torch.testing.assert_close(a.cpu().float(), b.float(), **_tol(dtype))


@pytest.mark.parametrize("n", [1, 640, 3 * 509])
def test_squashed_logits(n):
    x = torch.randn(3, n, generator=torch.Generator().manual_seed(n)) * 40.0
    want = host_ops.softcap_rows(x.clone(), 15.0)
    got = _ops().softcap_rows(x.cuda(), 15.0).cpu()
    torch.testing.assert_close(got, want, rtol=1e-5, atol=1e-5)
    assert float(got.abs().max()) <= 15.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [3, 130, 1500])
@pytest.mark.parametrize("E,k", [(2, 2), (16, 1), (60, 4), (130, 6)])
def test_sigmoid_router(dtype, T, E, k):
    g = torch.Generator().manual_seed(E + T)
    x = torch.randn(T, 64, generator=g).to(dtype)
    w = torch.randn(E, 64, generator=g) * 0.3
    tw, ti, _ = _ops().router_topk(x.cuda(), w.cuda(), k, False, 1.0, score="sigmoid")
    logits = x.double() @ w.double().T
    want, _ = torch.sort(torch.sigmoid(logits), dim=-1, descending=True)
    torch.testing.assert_close(tw.cpu(), want[:, :k].float(), rtol=1e-4, atol=1e-5)
    torch.testing.assert_close(torch.sigmoid(torch.gather(logits, 1, ti.cpu().long())).float(),
                               tw.cpu(), rtol=1e-4, atol=1e-5)
    assert all(len(set(r)) == k for r in ti.cpu().tolist())


def test_sigmoid_router_orders_saturated_scores_by_their_logits():
    """Scores that are all one in fp32 are still chosen by the larger logit."""
    E = 40
    w = torch.zeros(E, 32)
    w[:, 0] = torch.linspace(20.0, 60.0, E)[torch.randperm(E, generator=torch.Generator().manual_seed(1))]
    x = torch.zeros(200, 32)
    x[:, 0] = 1.0
    for rows in (4, 200):
        tw, ti, _ = _ops().router_topk(x[:rows].cuda(), w.cuda(), 3, False, 1.0, score="sigmoid")
        want = torch.topk(w[:, 0], 3).indices.tolist()
        assert all(r == want for r in ti.cpu().tolist()) and bool((tw == 1.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,k,H,I", [(1, 8, 2, 256, 64), (3, 6, 2, 64, 32), (40, 5, 3, 72, 40),
                                       (130, 4, 2, 128, 96), (700, 16, 1, 256, 64), (9, 3, 3, 45, 21)])
def test_weights_on_the_experts_inputs(dtype, T, E, k, H, I):
    """Dispatch with the weights of the grouped rows, gate/up product with a factor per row,
    plain sum of the experts' rows: every kernel that serves the product."""
    g = torch.Generator().manual_seed(T)
    ops = _ops()
    x = torch.randn(T, H, generator=g).to(dtype)
    gu = (torch.randn(E, 2 * I, H, generator=g) / math.sqrt(H) * 2.0).to(dtype)
    dn = (torch.randn(E, H, I, generator=g) / math.sqrt(I)).to(dtype)
    idx = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)]).to(torch.int32)
    tw = torch.rand(T, k, generator=g)
    ro, rr, rd, rw = host_ops.moe_dispatch(idx, E, topk_w=tw)
    do, dr, dd, dw = ops.moe_dispatch(idx.cuda(), E, topk_w=tw.cuda())
    for a, b in ((do, ro), (dr, rr), (dd, rd), (dw, rw)):
        assert torch.equal(a.cpu(), b)
    want = host_ops.grouped_gate_up_swiglu(x.float(), rr, ro, gu.float(), row_scale=rw)
    got = ops.grouped_gate_up_swiglu(x.cuda(), dr, do, gu.cuda(), row_scale=dw)
    torch.testing.assert_close(got.float().cpu(), want, **_tol(dtype))
    # the weight went in ahead of the activation, not behind it
    behind = host_ops.grouped_gate_up_swiglu(x.float(), rr, ro, gu.float()) * rw[:, None]
    assert float((behind - want).abs().max()) > 0.05
    forms = [lambda: ops.gemm_generic(x.cuda(), gu.cuda(), dr, do, dual=True,
                                      num_out_rows=T * k, row_scale=dw)]
    if dtype == torch.bfloat16 and H % 8 == 0:
        forms += [lambda: ops.gemm_small_m(x.cuda(), gu.cuda(), dr, do, True, T * k, row_scale=dw),
                  lambda: ops.gemm_small_m(x.cuda(), gu.cuda(), dr, do, True, T * k,
                                           rows_per_pass=16, row_scale=dw),
                  lambda: ops.grouped_gemm_tc(ops.gather_rows(x.cuda(), dr), do, gu.cuda(), True,
                                              row_scale=dw)]
        if H >= 256:
            forms += [lambda: ops.gemm_stream_grouped(x.cuda(), gu.cuda(), dr, do, True, T * k,
                                                      row_scale=dw)]
    for form in forms:
        torch.testing.assert_close(form().float().cpu(), want, **_tol(dtype))
    ops.check_async_errors()
    y = ops.grouped_down(got, do, dn.cuda())
    plain_sum = ops.moe_combine(y, dd, tw.cuda(), None, None, weighted=False).float().cpu()
    ref = torch.zeros(T, H)
    for s in range(k):
        ref += y.float().cpu()[rd.view(T, k)[:, s].long()]
    torch.testing.assert_close(plain_sum, ref, **_tol(dtype))
    gain = 1.0 + 0.1 * torch.randn(H, generator=g)
    for fn in (lambda r, p: ops.add_rmsnorm(r, p, gain.cuda(), 1e-5, dtype),
               lambda r, p: ops.add_rmsnorm_sum(r, [p], None, (gain.cuda(),), 1e-5, dtype)[0]):
        resid = torch.randn(T, H, generator=g)
        dev = resid.cuda()
        n = fn(dev, ops.moe_combine_pending(y, dd, tw.cuda(), None, None, weighted=False))
        torch.testing.assert_close(dev.cpu(), resid + ref, rtol=2e-2, atol=2e-2)
        torch.testing.assert_close(n.float().cpu(), host_ops.add_rmsnorm(
            (resid + ref).clone(), None, gain, 1e-5, torch.float32), rtol=3e-2, atol=3e-2)


def _forms(dtype, D, VD, page, ragged):
    tensor = dtype == torch.bfloat16 and D in (64, 128) and VD in (64, 128)
    if not ragged:
        return ["generic", "decode_any"] + (["decode"] if tensor else [])
    out = ["generic"]
    if D % 4 == 0 and VD % 4 == 0:
        out.append("tiled")
    if tensor:
        out.append("mma")
        if D == VD and page in (8, 16, 32, 64):
            out.append("tc")
    return out


def _distance(form, q, kc, vc, bt, step, scale, vec, chunk, VD, out_scale=1.0, lead=8):
    """One kernel form on views of columns; returns [T, heads * VD] on the host."""
    T, H = q.shape[0], vec[0].numel()
    wide = torch.full((T, lead + H * VD + 16), 5.0, dtype=q.dtype, device="cuda")
    out = wide[:, lead:lead + H * VD]
    _ops().distance_attention(_wide(q, lead, 24), kc.cuda(), vc.cuda(), bt.cuda(), _cuda(step),
                              scale, *[v.cuda() for v in vec], chunk, out, out_scale, kernel=form)
    _ops().check_async_errors()
    assert bool((wide[:, :lead] == 5).all()) and bool((wide[:, lead + H * VD:] == 5).all())
    return out.float().cpu()


def _reference(q, kc, vc, bt, step, scale, vec, chunk, VD, out_scale=1.0):
    return host_ops.distance_attention(q.float(), kc.float(), vc.float(), bt, step, scale, *vec,
                                       chunk, torch.empty(q.shape[0], vec[0].numel() * VD),
                                       out_scale)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,VD,page", [(6, 2, 16, 24, 4), (1, 1, 7, 9, 8), (8, 2, 64, 64, 16),
                                           (4, 4, 128, 128, 16), (16, 1, 64, 128, 16),
                                           (20, 1, 128, 64, 8), (3, 3, 64, 64, 64)])
@pytest.mark.parametrize("chunk", [0, 1, 33, 64, 100, 1000])
def test_distance_attention_of_portions(dtype, H, G, D, VD, page, chunk):
    """Ragged portions that start anywhere and cross the borders of runs, over pages of which
    those before the run were given back; every form that takes the sizes."""
    q_lens, starts = [5, 150, 2, 70], [96, 31, 199, 0]
    step, bt, kc, vc, q = _kv_case(H * D + chunk, H, G, D, VD, page, q_lens, starts, dtype, chunk)
    vec = _head_vectors(H, H)
    ref = _reference(q, kc, vc, bt, step, D ** -0.5, vec, chunk, VD, 0.7)
    for form in _forms(dtype, D, VD, page, True) + [None]:
        got = _distance(form, q, kc, vc, bt, step, D ** -0.5, vec, chunk, VD, 0.7)
        torch.testing.assert_close(got, ref, **_tol(dtype), msg=lambda m: f"{form}: {m}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,VD,page", [(6, 2, 16, 24, 4), (1, 1, 7, 9, 8), (8, 2, 64, 64, 16),
                                           (4, 4, 128, 128, 16), (16, 1, 64, 128, 16),
                                           (20, 1, 128, 64, 8)])
@pytest.mark.parametrize("chunk", [0, 1, 110, 500])
def test_distance_attention_of_single_tokens(dtype, H, G, D, VD, page, chunk):
    """One token a sequence at the first, last and inner places of runs, in splits."""
    starts = [0, 109, 110, 111, 999, 1000, 730]
    step, bt, kc, vc, q = _kv_case(H * D + chunk, H, G, D, VD, page, [1] * 7, starts, dtype, chunk)
    vec = _head_vectors(H, H + 1)
    ref = _reference(q, kc, vc, bt, step, D ** -0.5, vec, chunk, VD)
    for form in _forms(dtype, D, VD, page, False) + [None]:
        got = _distance(form, q, kc, vc, bt, step, D ** -0.5, vec, chunk, VD)
        torch.testing.assert_close(got, ref, **_tol(dtype), msg=lambda m: f"{form}: {m}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,VD", [(64, 64), (128, 64), (16, 24)])
def test_distance_attention_of_a_mixed_batch(dtype, D, VD):
    step, bt, kc, vc, q = _kv_case(3, 4, 2, D, VD, 16, [1, 1, 1, 40, 3], [50, 0, 129, 100, 62],
                                   dtype, 48)
    vec = _head_vectors(4, 9)
    ref = _reference(q, kc, vc, bt, step, 0.2, vec, 48, VD)
    got = _distance(None, q, kc, vc, bt, step, 0.2, vec, 48, VD)
    torch.testing.assert_close(got, ref, **_tol(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,VD", [(64, 64), (128, 128), (64, 128), (12, 8), (7, 9)])
@pytest.mark.parametrize("ragged", [True, False])
def test_a_run_s_first_key_is_seen_and_the_key_before_it_is_not(dtype, D, VD, ragged):
    """One key that outweighs all others, at the first place of the query's run, directly
    before it, at page borders and far back: the query's output is that key's value, or
    holds nothing of it.  The penalty is weak (a far key must still win)."""
    chunk, page = 110, 16
    for pos, key, seen in [(219, 110, True), (219, 109, False), (220, 219, False), (220, 220, True),
                           (221, 220, True), (1099, 990, True), (1099, 989, False),
                           (329, 256, True), (329, 255, True), (330, 0, False)]:
        n = 3 if ragged else 1
        start = pos - n + 1
        step, bt, kc, vc, q = _kv_case(7, 2, 1, D, VD, page, [n], [start], dtype)
        kc.mul_(0.05)
        q.mul_(0.05)
        u = torch.zeros(D)
        u[0] = 6.0
        at = (int(bt[0, key // page]), 0, key % page)
        kc[at] = u.to(dtype)
        q[n - 1] = u.repeat(2).to(dtype)
        vc[at] = 40.0
        vec = (torch.tensor([1.0, 1.5]), torch.tensor([0.3, 0.02]), torch.tensor([0.2, 0.1]))
        for form in _forms(dtype, D, VD, page, ragged):
            got = _distance(form, q, kc, vc, bt, step, 1.0, vec, chunk, VD)[n - 1]
            if seen:
                assert float((got - 40.0).abs().max()) < 0.5, (form, pos, key)
            else:
                assert float(got.abs().max()) < 10.0, (form, pos, key)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ragged", [True, False])
def test_the_penalty_decides_between_equal_keys(dtype, ragged):
    """All keys alike: the weights are the penalties' alone, (1 + r2 d)^(-r1) normalised, and a
    negative r1 prefers the far keys."""
    H, D, page, pos = 4, 64, 16, 300
    n = 2 if ragged else 1
    step, bt, kc, vc, q = _kv_case(5, H, 1, D, D, page, [n], [pos - n + 1], dtype)
    kc.fill_(0.25)
    q.fill_(0.5)
    vc.zero_()
    for p in range(pos + 1):
        vc[int(bt[0, p // page]), 0, p % page] = p / 64.0
    vec = (torch.tensor([1.0, 2.0, -1.0, 1.0]), torch.tensor([2.0, 0.5, -1.5, 0.0]),
           torch.tensor([0.7, 3.0, 0.5, 1.0]))
    d = torch.arange(pos, -1, -1, dtype=torch.float64)
    vals = vc[bt[0, torch.arange(pos + 1) // page].long(), 0, torch.arange(pos + 1) % page, 0].double()
    for form in _forms(dtype, D, D, page, ragged):
        got = _distance(form, q, kc, vc, bt, step, 0.1, vec, 0, D)[n - 1].view(H, D)
        for h in range(H):
            w = (1.0 + float(vec[2][h]) * d) ** (-float(vec[1][h]))
            want = float((w * vals).sum() / w.sum())
            tol = 2e-5 if dtype == torch.float32 else 6e-3
            assert float((got[h] - want).abs().max()) <= tol * max(1.0, abs(want)), (form, h)


def test_prompt_forms_do_not_depend_on_the_cut():
    """The tcgen05 and the tiled form walk key tiles at multiples of 64 of the absolute
    position.  The tiled form gives the same bits however a sequence was cut; in the tcgen05
    form a row's running reference moves with its warp's, which changes roundings only."""
    for dtype, form, D in ((torch.bfloat16, "tc", 128), (torch.float32, "tiled", 40)):
        step, bt, kc, vc, q = _kv_case(11, 4, 2, D, D, 16, [300], [0], dtype)
        vec = _head_vectors(4, 2)
        for chunk in (0, 90):
            whole = _distance(form, q, kc, vc, bt, step, 0.1, vec, chunk, D)
            for a, b in ((0, 37), (37, 164), (164, 166), (166, 300)):
                part = _distance(form, q[a:b], kc, vc, bt, _step([b - a], [a]), 0.1, vec, chunk, D)
                if form == "tiled":
                    assert torch.equal(part, whole[a:b]), (chunk, a)
                else:
                    torch.testing.assert_close(part, whole[a:b], rtol=8e-3, atol=1e-5)
                    assert float((part == whole[a:b]).float().mean()) > 0.98


@pytest.mark.parametrize("rank,dr", [(64, 16), (128, 32), (256, 64), (512, 64)])
@pytest.mark.parametrize("H", [4, 16, 70])
@pytest.mark.parametrize("q_lens,starts", [([1, 1, 1], [0, 700, 77]), ([1, 5, 90], [300, 2, 40])])
def test_latent_attention_with_16_bit_weights(rank, dr, H, q_lens, starts):
    """Two-term weights: closer to the fp32-arithmetic kernel than the 8-bit ones, and within
    one rounding of the result."""
    g = torch.Generator().manual_seed(rank + H)
    step = _step(q_lens, starts)
    page, S, T = 16, len(q_lens), sum(q_lens)
    need = [-(-(a + n) // page) for n, a in zip(q_lens, starts)]
    bt = torch.full((S, max(need)), -1, dtype=torch.int32)
    perm, at = torch.randperm(sum(need), generator=g).to(torch.int32), 0
    for s, n in enumerate(need):
        bt[s, :n] = perm[at:at + n]
        at += n
    cache = torch.randn(sum(need), 1, page, rank + dr, generator=g).bfloat16().cuda()
    q_lat = (torch.randn(H, T, rank, generator=g) * 0.4).bfloat16().cuda()
    q_rot = (torch.randn(T, H, dr, generator=g) * 0.4).bfloat16().cuda()
    st = _cuda(step)
    run = lambda **kw: _ops().latent_attention(q_lat, q_rot, cache, bt.cuda(), st, 0, 0.1, **kw)
    exact = _ops().latent_attention(q_lat.float(), q_rot.float(), cache.float(), bt.cuda(), st, 0,
                                    0.1, kernel="general").cpu()
    wide = run(kernel="mma", fp32_weights=True).float().cpu()
    narrow = run(kernel="mma").float().cpu()
    torch.testing.assert_close(wide, exact, rtol=5e-3, atol=1e-4)
    assert float((wide - exact).pow(2).mean()) <= float((narrow - exact).pow(2).mean())


# -- the engine ------------------------------------------------------------------------
def _folder_dtype(dtype):
    return "float32" if dtype == "float32" else "bfloat16"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,cfg,seed,lengths,page", CASES)
@pytest.mark.parametrize("kind", list(mc.TRACE_KINDS))
def test_replay_matches_plain(tmp_path, dtype, name, cfg, seed, lengths, page, kind):
    d = dk.make_model_dir(cfg, tmp_path / "m", seed, dtype=_folder_dtype(dtype))
    reqs = dk.make_requests(cfg, lengths, seed)
    ref = dk.reference_rows(d, reqs)
    steps = mc.TRACE_KINDS[kind](reqs)
    sess = ReplaySession(d, dtype, traces.peak_tokens(steps), page_size=page, max_live=4)
    rows = mc.run_trace(sess, steps)
    sess.executor.poll_errors()
    rows = dk.rows_to_compare(dtype, d, reqs, rows)
    mc.compare(rows, ref, dk.bound_for(dtype, d, reqs), f"{name}/{kind}/{dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_with_recorded_steps(tmp_path, dtype):
    """250 decoded tokens over many borders of two kinds of runs: pages before a run are given
    back and used again, the recurrences are carried through recorded steps."""
    cfg = dk.DA
    d = dk.make_model_dir(cfg, tmp_path / "m", 3, dtype=_folder_dtype(dtype))
    reqs = dk.make_requests(cfg, [270], 3)
    ref = dk.reference_rows(d, reqs)
    steps = traces.tail_decode(reqs, 250)
    sess = ReplaySession(d, dtype, traces.peak_tokens(steps), page_size=4, use_graphs=True)
    rows = mc.run_trace(sess, steps)
    assert len(rows) == 270 and sess.executor.graph_replays >= 200
    rows = dk.rows_to_compare(dtype, d, reqs, rows, share=0.03)
    mc.compare(rows, ref, dk.bound_for(dtype, d, reqs), f"long decode {dtype}")


@pytest.mark.parametrize("dtype,kind", [("bfloat16", "whole"), ("bfloat16", "mixed"),
                                        ("float32", "tail"), ("float32", "mixed")])
def test_long_prompts(tmp_path, dtype, kind):
    """Prompts of several hundred tokens at head sizes 48 to 128: many key tiles and runs, the
    recurrence in several stretches, attention over many pages."""
    cfg = dk.DD
    d = dk.make_model_dir(cfg, tmp_path / "m", 11, dtype=_folder_dtype(dtype))
    reqs = dk.make_requests(cfg, [700, 260], 11)
    ref = dk.reference_rows(d, reqs)
    steps = mc.TRACE_KINDS[kind](reqs)
    sess = ReplaySession(d, dtype, traces.peak_tokens(steps), page_size=16, max_live=4)
    rows = mc.run_trace(sess, steps)
    sess.executor.poll_errors()
    mc.compare(rows, ref, dk.bound_for(dtype, d, reqs), f"long/{kind}/{dtype}")


def test_prefill_equals_decoding_in_32_bit(tmp_path):
    """The same sequence whole, token by token and in portions of two: the three runs
    agree with each other far inside their distance to the plain model."""
    cfg = dk.DB
    d = dk.make_model_dir(cfg, tmp_path / "m", 6)
    reqs = dk.make_requests(cfg, [75], 6)
    runs = []
    for steps in (traces.whole(reqs), traces.tail_decode(reqs, 74),
                  traces.portions(reqs, sizes=(2,))):
        sess = ReplaySession(d, "float32", 128, page_size=8, max_live=1)
        rows = mc.run_trace(sess, steps)
        runs.append(torch.stack([rows[("r0", p)] for p in range(75)]))
    scale = float(runs[0].abs().max())
    for other in runs[1:]:
        assert float((other - runs[0]).abs().max()) / scale < 2e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_equals_each_alone(tmp_path, dtype):
    """Four requests of unequal lengths in one step, and then a token of each, against each
    alone in a pool whose pages and slots other requests have used."""
    cfg = dk.DD
    d = dk.make_model_dir(cfg, tmp_path / "m", 8, dtype=_folder_dtype(dtype))
    reqs = dk.make_requests(cfg, [70, 3, 131, 48], 8)

    def steps(groups):
        out = []
        for ids in groups:
            for part in (slice(0, -1), slice(-1, None)):
                out.append({"step": len(out), "end": ids if part.start == -1 else [],
                            "entries": [{"id": r, "tokens": reqs[r][part],
                                         "want": [len(reqs[r][part]) - 1]} for r in ids]})
        return out
    results = []
    for groups in ([list(reqs)], [[r] for r in reqs]):
        sess = ReplaySession(d, dtype, 320, page_size=16, max_live=4)
        results.append(mc.run_trace(sess, steps(groups)))
    bound = 2e-5 if dtype == "float32" else dk.bound_for(dtype, d, reqs)
    mc.compare(results[1], results[0], bound, "alone")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(tmp_path, dtype):
    cfg = dk.DA
    d = dk.make_model_dir(cfg, tmp_path / "m", 5, dtype="bfloat16")
    reqs = dk.make_requests(cfg, [70, 33, 20, 9, 50, 41], 5)
    ref = dk.reference_rows(d, reqs)
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
    rows = dk.rows_to_compare(dtype, d, reqs, traces.collect(steps, outs), share=0.1)
    mc.compare(rows, ref, dk.bound_for(dtype, d, reqs), f"trace_run/{dtype}")


def test_greedy_generation_through_the_engine(tmp_path):
    from inferx_b200 import Engine, EngineConfig, Request, SamplingParams
    d = dk.make_model_dir(dk.DA, tmp_path / "m", 4)
    c, w = plain.read_model_folder(d)
    prompts = list(dk.make_requests(dk.DA, [7, 19, 3, 30, 11], 8).values())
    eng = Engine.create(EngineConfig(model=d, dtype="float32", block_size=4, max_num_seqs=3,
                                     num_gpu_blocks_override=96, prefill_chunk=6,
                                     max_model_len=64))
    done = eng.generate([Request(p, SamplingParams(max_tokens=12, ignore_eos=True))
                         for p in prompts])
    for p, c_out in zip(prompts, done):
        seq = list(p)
        for tok in c_out.output_tokens:
            lg = plain.forward(c, w, seq)[-1]
            top = torch.topk(lg, 2).values
            # the engine's choice is the plain model's, unless the two best are a tie in fp32
            assert tok == int(lg.argmax()) or float(top[0] - top[1]) < 1e-4 * float(lg.abs().max())
            seq.append(tok)
        assert len(c_out.output_tokens) == 12


def test_command_line(tmp_path):
    """The generation program takes a folder of the design like any other: greedy output is
    the plain model's, and sampling with a seed gives the same tokens twice."""
    d = dk.make_model_dir(dk.DB, tmp_path / "m", 9)
    c, w = plain.read_model_folder(d)
    base = [sys.executable, os.path.join(ROOT, "bin", "inferx-generate"), d, "--dtype", "fp32",
            "--block-size", "4", "--max-model-len", "64", "--max-num-seqs", "2",
            "--num-gpu-blocks-override", "48", "--log-level", "warning", "--ignore-eos"]

    def run(*args):
        p = subprocess.run(base + list(args), capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        return [json.loads(ln)["output_ids"] for ln in p.stdout.splitlines() if ln.startswith("{")]
    outs = run("--prompt-ids", "5,17,3,80,41", "--prompt-ids", "9 8 7", "--max-tokens", "6")
    for ids, prompt in zip(outs, ([5, 17, 3, 80, 41], [9, 8, 7])):
        seq = list(prompt)
        for tok in ids:
            lg = plain.forward(c, w, seq)[-1]
            top = torch.topk(lg, 2).values
            assert tok == int(lg.argmax()) or float(top[0] - top[1]) < 1e-4 * float(lg.abs().max())
            seq.append(tok)
        assert len(ids) == 6
    sampled = [run("--prompt-ids", "9 8 7", "--max-tokens", "8", "--temperature", "0.9", "--top-k",
                   "20", "--top-p", "0.9", "--seed", "3") for _ in range(2)]
    assert sampled[0] == sampled[1] and len(sampled[0][0]) == 8

"""Tatelorn on the GPU.  Each new kernel alone against the plain functions of tests/plain_tatelorn.py (the stream's start: token row,
position row, norm; a normalised addend without a norm behind it; gated activations on their own rows and inside the products;
normed heads, mixed values and the cache write; capped attention with a sink of score 0 and a stand-out key far back, at page and
tile borders and at the query itself, as rows of a portion and as decoded tokens, with scores inside half the cap, up to it and far
beyond it, through the general kernel, the mma.sync kernels with their merges, the fused decode kernel and the tcgen05 kernel; the
router, the clamped experts and the shared one); then whole models under every way of cutting the work, in 32-bit and in bfloat16;
greedy generation through the engine's entry point with and without CUDA graphs; the trace runner as a program."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from helpers import max_error, random_tokens, replay_and_collect, trace_mixed, trace_portions, trace_tail, trace_whole
import plain_tatelorn as plain
from tatelorn_cases import BLOCK_SIZE, CONFIGS, owed, plain_logits, rounded_plain, write_case

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


def K():
    from iian_b200 import ops
    return ops.kernels()


def launched(before):
    from iian_b200.ops import cuda_backend
    return {k: v - before.get(k, 0) for k, v in cuda_backend.LAUNCHES_BY_ENTRY.items() if v != before.get(k, 0)}


def launches():
    from iian_b200.ops import cuda_backend
    return dict(cuda_backend.LAUNCHES_BY_ENTRY)


def close(got, want, dtype, what, rel16=2e-2, abs32=2e-5):
    got, want = got.double().cpu(), want.double().cpu()
    tol = abs32 * max(1.0, want.abs().max().item()) if dtype == "float32" else rel16 * want.abs().max().item()
    err = (got - want).abs().max().item()
    assert err <= tol, f"{what} [{dtype}]: max error {err:.3g} > {tol:.3g}"


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# ---- row-wise kernels ---------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n, h", [(5, 72), (3, 100), (4, 1000), (2, 4100), (3, 30), (700, 128), (2000, 260)])
def test_where_the_stream_starts(dtype, n, h):
    g = torch.Generator().manual_seed(h)
    V, P = 41, 90
    table, places = torch.randn(V, h, generator=g).to(DT[dtype]), (torch.randn(P, h, generator=g) * 2).to(DT[dtype])
    w = torch.randn(h, generator=g) * 0.3
    toks, pos = torch.randint(0, V, (n,), generator=g), torch.randint(0, P, (n,), generator=g)
    toks[0], pos[0], pos[-1] = V - 1, P - 1, 0
    for with_places, with_norm, with_copy in ((1, 1, 1), (1, 1, 0), (0, 1, 1), (1, 0, 1), (0, 0, 1)):
        x = torch.empty(n, h, device=DEV)
        copy = torch.empty(n, h, device=DEV, dtype=DT[dtype]) if with_copy else None
        K().embedding_placed(table.to(DEV), toks.int().to(DEV), 3.25, places.to(DEV) if with_places else None, pos.int().to(DEV),
                             (1 + w).to(DEV) if with_norm else None, 1e-5, x, copy)
        want = table.double()[toks] * 3.25
        if with_places:
            want = want + places.double()[pos]
        if with_norm:
            want = plain.centred_norm(want, w.double(), 1e-5)
        close(x, want, "float32", f"stream of width {h}")
        if with_copy:
            assert torch.equal(copy, x.to(DT[dtype]))
    # a padding token (position -1) reads inside the tables
    K().embedding_placed(table.to(DEV), i32([0]), 1.0, places.to(DEV), i32([-1]), None, 0.0, torch.empty(1, h, device=DEV), None)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n, h", [(5, 72), (3, 101), (2, 4100), (900, 128)])
def test_a_normalised_addend_and_the_stream_itself(dtype, n, h):
    g = torch.Generator().manual_seed(h)
    x, y = torch.randn(n, h, generator=g) * 3, (torch.randn(n, h, generator=g) * 7).to(DT[dtype])
    u = torch.randn(h, generator=g)
    for with_y, with_u, with_out in ((1, 1, 1), (1, 1, 0), (1, 0, 1), (0, 0, 1)):
        res = x.to(DEV).clone()
        out = torch.empty(n, h, device=DEV, dtype=DT[dtype]) if with_out else None
        K().normed_add_rms_norm(res, y.to(DEV) if with_y else None, u.to(DEV) if with_u else None, 1e-5, None, None, 0.0, out)
        want = x.double()
        if with_y:
            want = want + (plain.over_rms(y.double(), 1e-5) * u.double() if with_u else y.double())
        close(res, want, "float32", f"stream of width {h}")
        if with_out:
            assert torch.equal(out, res.to(DT[dtype]))


def _gated(g, u, activation, limit):
    if activation == "relu":
        return torch.relu(g) * u
    if activation == "silu":
        return g * torch.sigmoid(g) * u
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("activation, limit", [("relu", 0.0), ("clamped_swish", 0.7), ("silu", 0.0)])
def test_gated_activations_on_rows_and_inside_products(dtype, activation, limit):
    g = torch.Generator().manual_seed(3)
    for n, F in ((3, 40), (5, 44), (130, 64)):
        wide = (torch.randn(n, 2 * F + 8, generator=g) * 2).to(DT[dtype])
        out = torch.empty(n, F, device=DEV, dtype=DT[dtype])
        inter = 8 if F % 8 == 0 else 0
        K().gated_act(wide.to(DEV)[:, : 2 * F], out, inter, activation, limit)
        v = wide.double()[:, : 2 * F]
        gate, up = (v.view(n, F // 8, 2, 8)[:, :, 0].reshape(n, F), v.view(n, F // 8, 2, 8)[:, :, 1].reshape(n, F)) if inter else (v[:, :F], v[:, F:])
        close(out, _gated(gate, up, activation, limit), dtype, f"{activation} of {n} x {F}", rel16=8e-3)
    if dtype == "float32":
        return
    for n, F, W, entry in ((1, 64, 96, "gemm_stream_gated"), (8, 128, 320, "gemm_stream_gated"), (130, 96, 128, "gemm_tcgen05_gated"),
                           (300, 256, 200, "gemm_tcgen05_gated"), (700, 320, 64, "gemm_tcgen05_gated")):
        x = torch.randn(n, W, generator=g).to(torch.bfloat16)
        w = (torch.randn(2 * F, W, generator=g) * 0.3).to(torch.bfloat16)
        assert K().can_fuse_gated(x.to(DEV), w.to(DEV), 8, activation)
        before = launches()
        out = torch.empty(n, F, device=DEV, dtype=torch.bfloat16)
        K().linear_gated(x.to(DEV), w.to(DEV), out, activation, limit)
        K().check_device_status()
        assert entry in launched(before)
        v = (x.double() @ w.double().T).view(n, F // 8, 2, 8)
        close(out, _gated(v[:, :, 0].reshape(n, F), v[:, :, 1].reshape(n, F), activation, limit), dtype, f"{activation} in {entry}", rel16=8e-3)


# ---- normed heads, mixed values, cache write ----------------------------------------------------------------
def _fill_cache(dtype, H, G, d, dv, n, page, seed, share=0.0, extra=8, weights=True, eps=1e-5):
    """Projections of n tokens of one sequence through the kernel into a paged cache of scattered pages; returns what the plain
    functions make of the same rows."""
    g = torch.Generator().manual_seed(seed)
    nq, nk, nv = H * d, G * d, G * dv
    proj = torch.randn(n, nq + nk + nv + extra, generator=g).to(DT[dtype])               # the mixer's columns start behind `extra` others
    first = torch.randn(n, nv + 16, generator=g).to(DT[dtype])
    qn, kn = (0.5 + torch.rand(d, generator=g) for _ in range(2))
    n_used = -(-n // page)
    order = torch.randperm(n_used + 3, generator=g)[:n_used].to(torch.int32)
    kc = torch.zeros(n_used + 3, G, page, d, dtype=DT[dtype], device=DEV)
    vc = torch.zeros(n_used + 3, G, page, dv, dtype=DT[dtype], device=DEV)
    pos = torch.arange(n, dtype=torch.int32)
    slots = (order[(pos // page).long()] * page + pos % page).to(torch.int32)
    q = torch.empty(n, H, d, dtype=DT[dtype], device=DEV)
    K().head_norm_store(proj.to(DEV)[:, extra:], 0, nq, nq + nk, q, kc, vc, slots.to(DEV), num_heads=H, num_kv_heads=G, k_dim=d, v_dim=dv,
                        q_weight=qn.to(DEV) if weights else None, k_weight=kn.to(DEV) if weights else None, eps=eps,
                        first_values=first.to(DEV)[:, 16:] if share else None, share=share)
    p = proj.double()[:, extra:]
    qw, kw = p[:, :nq].reshape(n, H, d), p[:, nq:nq + nk].reshape(n, G, d)
    if weights:
        qw, kw = plain.over_rms(qw, eps) * qn.double(), plain.over_rms(kw, eps) * kn.double()
    vw = plain.mixed_values(p[:, nq + nk:].reshape(n, G, dv), first.double()[:, 16:].reshape(n, G, dv) if share else None, share)
    return SimpleNamespace(proj=proj, first=first, qn=qn, kn=kn, q=q, kc=kc, vc=vc, order=order, slots=slots, pos=pos, q_want=qw, k_want=kw,
                           v_want=vw, eps=eps)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, d, dv", [(6, 2, 16, 24), (3, 3, 40, 24), (2, 1, 128, 128), (8, 2, 64, 64), (1, 1, 22, 7), (5, 1, 200, 8), (2, 1, 8, 320),
                                         (1, 1, 512, 512), (4, 2, 64, 128)])
@pytest.mark.parametrize("share", [0.0, 0.375, -0.25])
def test_normed_heads_mixed_values_and_cache_write(dtype, H, G, d, dv, share):
    for n, weights in ((5, True), (70, True), (9, False)):
        c = _fill_cache(dtype, H, G, d, dv, n, 8, seed=d + n, share=share, weights=weights)
        close(c.q, c.q_want, dtype, "normed queries", rel16=1e-2)
        cells = c.slots.long().to(DEV)
        close(c.kc.permute(0, 2, 1, 3).reshape(-1, G, d)[cells], c.k_want, dtype, "keys in their cells", rel16=1e-2)
        close(c.vc.permute(0, 2, 1, 3).reshape(-1, G, dv)[cells], c.v_want, dtype, "values in their cells", rel16=8e-3)
        assert int((c.kc != 0).any(-1).any(1).sum()) == n, "cells of other tokens were written"
        # a padding token (cell -1) stores nothing, and nothing is written beyond the cache
        kb, vb = c.kc.clone(), c.vc.clone()
        cells = c.kc.shape[0] * 8
        K().head_norm_store(torch.randn(2, H * d + G * (d + dv), device=DEV).to(DT[dtype]), 0, H * d, (H + G) * d,
                            torch.empty(2, H, d, device=DEV, dtype=DT[dtype]), c.kc, c.vc, i32([-1, cells]), num_heads=H, num_kv_heads=G,
                            k_dim=d, v_dim=dv, q_weight=c.qn.to(DEV), k_weight=c.kn.to(DEV), eps=1e-5)
        assert torch.equal(kb, c.kc) and torch.equal(vb, c.vc)


# ---- attention ---------------------------------------------------------------------------------------------
def _meta(c_pos, rows, bt, decode_only=False, slots=None):
    r = torch.tensor(rows)
    return SimpleNamespace(positions=c_pos[r].to(DEV), seq_of_token=torch.zeros(len(rows), dtype=torch.int32, device=DEV),
                           cu_q=i32([0, len(rows)]), ctx_len=i32([rows[-1] + 1]), block_table=bt.to(DEV), num_seqs=1, num_tokens=len(rows),
                           max_q_len=len(rows), max_ctx=rows[-1] + 1, decode_only=decode_only, slots=slots)


ATTENTION = [  # H, G, d, dv, page, n, cap, strength: what the stand-out scores come to before the cap
    (6, 2, 16, 24, 16, 300, 6.0, 9.0), (4, 4, 64, 64, 8, 300, 20.0, 9.0), (8, 2, 64, 64, 16, 700, 10.0, 30.0), (3, 1, 24, 8, 16, 150, None, 8.0),
    (4, 1, 128, 128, 32, 1500, 30.0, 12.0), (4, 2, 128, 128, 16, 2600, 14.0, 12.0), (2, 2, 40, 200, 16, 260, 15.0, 9.0), (5, 1, 22, 12, 8, 90, 9.0, 8.0),
    (32, 1, 128, 128, 64, 400, 8.0, 25.0), (6, 3, 128, 128, 24, 200, 12.0, 9.0), (4, 1, 64, 64, 16, 1300, None, 10.0), (8, 1, 128, 128, 16, 300, None, 9.0),
    (6, 1, 128, 128, 128, 900, 40.0, 9.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, d, dv, page, n, cap, strength", ATTENTION)
def test_capped_attention_with_a_fixed_sink(dtype, H, G, d, dv, page, n, cap, strength):
    """Keys are made to stand out by putting a multiple of a query into their cells: far back, at a page's and a tile's last and first
    place, the query's own position.  Queries: a portion of the last 7 tokens, the same one by one (keys in one part and in several),
    the first ones, long portions.  Heads of 64 or 128 run on the tensor-core kernels in bfloat16, each with the score's bound told
    and not told."""
    c = _fill_cache(dtype, H, G, d, dv, n, page, seed=H * d)
    head0 = torch.arange(G) * (H // G)
    cut = 256 if page == 128 else 128 if n > 160 else 32
    marks = [(1, n - 1), (2, n - 2), (cut - 1, n - 3), (cut, n - 4), (page - 1, n - 5), (page, n - 6), (n - 7, n - 7)]
    scale = 0.3 / d ** 0.5
    for j, asker in marks:
        aq = c.q_want[asker, head0]
        key = (aq * (strength / scale / (aq * aq).sum(-1, keepdim=True))).to(DT[dtype])          # its score is `strength`
        cell = int(c.slots[j])
        c.kc[cell // page, :, cell % page] = key.to(DEV)
        c.k_want[j] = key.double()
    want = plain.grouped_attention(c.q_want, c.k_want, c.v_want, scale, cap).reshape(n, H * dv)
    bent = (lambda s: cap * torch.tanh(s / cap)) if cap else (lambda s: s)
    scores = torch.einsum("ihd,jhd->hij", c.q_want, c.k_want[:, torch.arange(H) // (H // G)]) * scale
    for j, asker in marks:                                                                       # without its key a row is another one
        e = torch.exp(bent(scores[0, asker, : asker + 1]))
        assert e[j] / (1 + e.sum()) > (0.1 if n < 1000 else 0.02), "the stand-out key must matter"
    no_sink = torch.exp(bent(scores[0, 0, :1])).sum()
    assert 1 / (1 + no_sink) > 0.2, "the sink must matter to the first token"
    if cap and strength > cap / 2:
        uncapped = plain.grouped_attention(c.q_want[n - 7:], c.k_want, c.v_want, scale, None, n - 7).reshape(7, H * dv)
        assert (uncapped - want[n - 7:]).abs().max() > 5e-3, "the cap must show"
    bound = 1.02 * scores.abs().max().item()
    bt = torch.full((1, max(64, c.order.numel())), -1, dtype=torch.int32)
    bt[0, : c.order.numel()] = c.order
    sink = torch.zeros(H, device=DEV)
    before = launches()
    for rows in (list(range(n - 7, n)), [n - 4], [n - 3], [n - 2], [n - 1], [0], list(range(0, 3)), list(range(max(0, n - 200), n)),
                 list(range(0, min(n, 130))), list(range(cut - 1, cut + 2))):
        r = torch.tensor(rows)
        meta = _meta(c.pos, rows, bt)
        variants = [(None, 0.0), (None, bound)] if cap else [(None, 0.0)]
        if len(rows) == 1:
            variants += [(split, 0.0) for split in (1, 2, 4, 8, 16)]
        for split, b in variants:
            out = torch.empty(len(rows), H * dv, dtype=DT[dtype], device=DEV)
            K().window_attention(c.q[r.to(DEV)].reshape(len(rows), H * d), c.kc, c.vc, out, meta, num_heads=H, num_kv_heads=G, k_dim=d, v_dim=dv,
                                 scale=scale, window=None, keep_first=0, sink=sink, gate=None, gate_per_head=True, n_split=split, softcap=cap,
                                 score_bound=b)
            close(out, want[r], dtype, f"rows {rows[0]}..{rows[-1]}, parts {split}, bound {b:.3g}", rel16=2.5e-2)
    K().check_device_status()
    ran = launched(before)
    fast = dtype == "bfloat16" and d == dv and d in (64, 128)
    assert ("window_attention" in ran) != fast, f"which kernel served it: {ran}"
    if fast:
        tc = "capped attention (tcgen05)" if cap else "chunked attention (tcgen05)"
        assert ("capped attention (mma)" if cap else "chunked attention (mma)") in ran and (tc in ran) == (d == 128 and page in (8, 16, 32, 64, 128)), ran


def test_capped_attention_keeps_windows():
    """The cap together with a window (another design's use of the parts): the general kernel in 32-bit, mma.sync and tcgen05."""
    for dtype, d in (("float32", 24), ("bfloat16", 64), ("bfloat16", 128)):
        H, G, n, page, window, cap = 4, 2, 420, 16, 150, 5.0
        c = _fill_cache(dtype, H, G, d, d, n, page, seed=d)
        scale = 4.0 / d ** 0.5
        bt = torch.full((1, 64), -1, dtype=torch.int32)
        bt[0, : c.order.numel()] = c.order
        for rows in ([n - 1], list(range(n - 60, n)), list(range(0, 200))):
            out = torch.empty(len(rows), H * d, dtype=DT[dtype], device=DEV)
            r = torch.tensor(rows)
            K().window_attention(c.q[r.to(DEV)].reshape(len(rows), H * d), c.kc, c.vc, out, _meta(c.pos, rows, bt), num_heads=H, num_kv_heads=G,
                                 k_dim=d, v_dim=d, scale=scale, window=window, keep_first=0, sink=torch.zeros(H, device=DEV), gate=None,
                                 gate_per_head=True, softcap=cap, score_bound=0.0)
            for k in (0, len(rows) - 1):
                i = rows[k]
                lo = max(0, i - window + 1)
                want = plain.grouped_attention(c.q_want[i:i + 1], c.k_want[lo:i + 1], c.v_want[lo:i + 1], scale, cap, i - lo).reshape(H * d)
                close(out[k], want, dtype, f"row {i} behind a window", rel16=2.5e-2)
        K().check_device_status()


@pytest.mark.parametrize("H, G, d, cap, share", [(8, 2, 64, 9.0, 0.375), (4, 1, 128, 30.0, 0.6875), (16, 1, 128, 4.0, -0.25), (4, 4, 64, None, 0.5), (6, 2, 128, 12.0, 0.0)])
def test_norms_mix_write_and_attention_of_decoded_tokens_in_one_kernel(H, G, d, cap, share):
    """Steps of one token per sequence, unequal contexts, one padding sequence: the kernel's output, the key and the value it leaves in
    the cell, and that both bits are those of the separate kernels."""
    from iian_b200.ops import cuda_backend
    g = torch.Generator().manual_seed(d + H)
    for lengths in ([1, 2, 17, 700], [5] * 40, [1500]):
        S, page = len(lengths), 16
        n_pages = sum(-(-n // page) for n in lengths)
        order = torch.randperm(n_pages, generator=g).to(torch.int32)
        kc = torch.randn(n_pages, G, page, d, generator=g).to(torch.bfloat16)
        vc = torch.randn(n_pages, G, page, d, generator=g).to(torch.bfloat16)
        bt = torch.full((S + 1, 128), -1, dtype=torch.int32)
        slots, ks = [], 0
        for s, n in enumerate(lengths):
            k = -(-n // page)
            bt[s, :k] = order[ks:ks + k]
            slots.append(int(order[ks + (n - 1) // page]) * page + (n - 1) % page)
            ks += k
        proj = torch.randn(S + 1, (H + 2 * G) * d, generator=g).to(torch.bfloat16)
        first = torch.randn(S + 1, G * d + 8, generator=g).to(torch.bfloat16)
        qn, kn = (0.5 + torch.rand(d, generator=g) for _ in range(2))
        meta = SimpleNamespace(positions=i32([n - 1 for n in lengths] + [0]), seq_of_token=i32(list(range(S)) + [-1]), cu_q=i32(list(range(S + 2))),
                               ctx_len=i32(lengths + [1]), block_table=bt.to(DEV), num_seqs=S + 1, num_tokens=S + 1, max_q_len=1,
                               max_ctx=max(lengths), decode_only=True, slots=i32(slots + [-1]))
        scale = 0.5
        sink = torch.zeros(H, device=DEV)
        kw = dict(num_heads=H, num_kv_heads=G)
        fv = first.to(DEV)[:, 8:] if share else None
        kc1, vc1, out = kc.to(DEV), vc.to(DEV), torch.empty(S + 1, H * d, dtype=torch.bfloat16, device=DEV)
        assert K().can_fuse_decode_attention(proj.to(DEV), meta, head_dim=d, rot_dim=0, rope_style=0, bias=None, **kw)
        K().attention_decode_fused(proj.to(DEV), kc1, vc1, out, meta, head_dim=d, scale=scale, window=None, q_weight=qn.to(DEV), k_weight=kn.to(DEV),
                                   eps=1e-5, table=None, slots=meta.slots, write_kv=True, sink=sink, softcap=cap, first_values=fv, share=share, **kw)
        kc2, vc2, q = kc.to(DEV), vc.to(DEV), torch.empty(S + 1, H, d, dtype=torch.bfloat16, device=DEV)
        K().head_norm_store(proj.to(DEV), 0, H * d, (H + G) * d, q, kc2, vc2, meta.slots, k_dim=d, v_dim=d, q_weight=qn.to(DEV), k_weight=kn.to(DEV),
                            eps=1e-5, first_values=fv, share=share, **kw)
        K().check_device_status()
        assert torch.equal(vc1, vc2), "the mixed value has one rounding, whichever kernel stores it"
        assert ((kc1.double() - kc2.double()).abs().max() / kc2.double().abs().max()) < 5e-3
        p = proj.double()
        for s, n in list(enumerate(lengths))[:4]:
            js = torch.arange(n)
            kk, vv = kc.double()[bt[s, js // page].long(), :, js % page], vc.double()[bt[s, js // page].long(), :, js % page]
            kk[n - 1] = plain.over_rms(p[s, H * d:(H + G) * d].view(G, d), 1e-5) * kn.double()
            vv[n - 1] = plain.mixed_values(p[s, (H + G) * d:].view(G, d), first.double()[s, 8:].view(G, d) if share else None, share)
            qq = plain.over_rms(p[s, : H * d].view(1, H, d), 1e-5) * qn.double()
            want = plain.grouped_attention(qq, kk, vv, scale, cap, n - 1).reshape(H * d)
            close(out[s], want, "bfloat16", f"sequence {s} of {n} keys", rel16=2.5e-2)


@pytest.mark.parametrize("G, rep, d, lengths", [(2, 3, 128, [1, 70, 500, 33, 64, 65]), (8, 4, 128, [900, 2, 128, 1]), (1, 16, 64, [300] * 40),
                                                (2, 4, 64, [400, 1, 63, 64, 65])])
def test_capped_attention_batches(G, rep, d, lengths):
    """Several sequences in one launch (decoded tokens beside portions, a padding sequence, many sequences: the TMA form)."""
    H, page = G * rep, 16
    for scale, cap, tell in ((0.02, 30.0, True), (0.3, 50.0, False), (0.6, 9.0, False)):
        for tail in (1, 5, 40):
            g = torch.Generator().manual_seed(tail)
            S = len(lengths)
            n_pages = sum(-(-n // page) for n in lengths)
            order = torch.randperm(n_pages, generator=g).to(torch.int32)
            kc = torch.randn(n_pages, G, page, d, generator=g).to(torch.bfloat16)
            vc = torch.randn(n_pages, G, page, d, generator=g).to(torch.bfloat16)
            bt = torch.full((S + 1, 64), -1, dtype=torch.int32)
            cu, pos, seq, ks = [0], [], [], 0
            for s, n in enumerate(lengths):
                k = -(-n // page)
                bt[s, :k] = order[ks:ks + k]
                ks += k
                t = min(tail, n)
                pos += list(range(n - t, n))
                seq += [s] * t
                cu.append(cu[-1] + t)
            cu.append(cu[-1] + 1)                              # a padding sequence: one token, no pages
            pos.append(0)
            seq.append(-1)
            q = torch.randn(cu[-1], H * d, generator=g).to(torch.bfloat16)
            meta = SimpleNamespace(positions=i32(pos), seq_of_token=i32(seq), cu_q=i32(cu), ctx_len=i32(lengths + [1]), block_table=bt.to(DEV),
                                   num_seqs=S + 1, num_tokens=cu[-1], max_q_len=min(tail, max(lengths)), max_ctx=max(lengths))
            out = torch.empty(cu[-1], H * d, dtype=torch.bfloat16, device=DEV)
            K().window_attention(q.to(DEV), kc.to(DEV), vc.to(DEV), out, meta, num_heads=H, num_kv_heads=G, k_dim=d, v_dim=d, scale=scale,
                                 window=None, keep_first=0, sink=torch.zeros(H, device=DEV), gate=None, gate_per_head=True, softcap=cap,
                                 score_bound=scale * 7.0 * d ** 0.5 if tell else 0.0)
            K().check_device_status()
            for s, n in enumerate(lengths[:6]):
                js = torch.arange(n)
                cells = bt[s, js // page].long(), js % page
                a, b = cu[s], cu[s + 1]
                want = plain.grouped_attention(q.double()[a:b].view(b - a, H, d), kc.double()[cells[0], :, cells[1]],
                                               vc.double()[cells[0], :, cells[1]], scale, cap, n - (b - a))
                close(out[a:b], want.reshape(b - a, H * d), "bfloat16", f"sequence {s} of {n} keys, {b - a} rows", rel16=2.5e-2)


# ---- experts ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n, experts, top, width, ff, limit, shared", [
    (1, 3, 1, 64, 32, 0.5, (16, 0.2)), (9, 5, 2, 96, 48, 1.5, None), (300, 8, 3, 128, 64, 0.8, (96, 1.7)), (40, 2, 2, 100, 36, 1.0, (20, 0.4)),
    (17, 30, 4, 64, 24, 2.0, (24, 0.3)), (5, 1, 1, 72, 40, 0.6, (8, 5.0)), (600, 12, 2, 256, 128, 1.2, (128, 0.5)), (8, 6, 2, 320, 64, 1.1, (64, 0.9))])
def test_router_clamped_experts_and_the_shared_one(dtype, n, experts, top, width, ff, limit, shared):
    from iian_b200.config.spec import PartSpec
    from iian_b200.engine.runner import StepContext, Workspace
    from iian_b200.parts.experts import RoutedExperts
    g = torch.Generator().manual_seed(n + experts)
    part = RoutedExperts(PartSpec("routed_experts", {
        "hidden_size": width, "num_experts": experts, "top": top, "intermediate_size": ff, "activation": "clamped_swish", "limit": limit,
        "score": "softmax_top", "router_bias": False, "weight_on": "output", "shared_intermediate_size": shared[0] if shared else 0,
        "shared_limit": shared[1] if shared else 0.0, "shared_gate": True}), DT[dtype], torch.device(DEV))
    tensors = {name: (torch.randn(*ts.shape, generator=g) * (0.2 if name in ("router", "shared.sg") else 0.15)).to(DT[dtype])
               for name, ts in part.tensors().items()}
    assert "router.b" not in tensors and ("shared.sg" in tensors) == bool(shared)
    part.bind({k: v.to(DEV) for k, v in tensors.items()})
    h = torch.randn(n, width, generator=g).to(DT[dtype])
    out = part.forward(h.to(DEV), StepContext(Workspace(torch.device(DEV))))
    K().check_device_status()
    w64 = {k: v.double() for k, v in tensors.items()}
    cfg = {"router": {"experts": experts, "top": top}, "expert": {"limit": limit}, "shared": {"limit": shared[1]} if shared else None}
    plain.router_margins = []
    try:
        want = plain.experts_feed_forward(cfg, w64, "", h.double())
        margins = plain.router_margins[0]
    finally:
        plain.router_margins = None
    if shared and shared[1] != limit:
        other = plain.experts_feed_forward(dict(cfg, shared={"limit": limit}), w64, "", h.double())
        assert (other - want).abs().max() > 1e-3, "the shared expert's own limit must show"
    safe = margins > (1e-6 if dtype == "float32" else 2e-2)            # rows where rounding cannot change the choice
    assert safe.sum() > 0.6 * n
    close(out[safe.to(DEV)], want[safe], dtype, "experts' weighted sum and the shared expert", rel16=3e-2, abs32=3e-5)


# ---- whole models --------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("tatelorn_gpu")
    out = {(name, "float32"): write_case(root, name) for name in CONFIGS}
    out.update({(name, "bfloat16"): write_case(root, name, steady=True) for name in CONFIGS})     # see steady_routers
    return out


LENGTHS = {"K": [1, 9, 40, 75, 130], "L": [3, 35, 70, 20, 100], "M": [2, 90, 33, 150], "N": [70, 5, 120, 33], "R": [41, 3, 77]}
_plain_cache = {}


def requests_and_plain(folders, name, dtype, lengths=None, seed=40, folder=None, reqs=None):
    folder = folder or folders[(name, dtype)]
    key = (folder, tuple(lengths or LENGTHS[name]), seed)
    if key not in _plain_cache:
        if reqs is None:
            reqs = {f"r{i}": random_tokens(CONFIGS[name]["vocab"], n, seed + i) for i, n in enumerate(lengths or LENGTHS[name])}
        _plain_cache[key] = (reqs, (plain_logits(folder, reqs), {dtype: rounded_plain(folder, reqs, DT[dtype])}))
    return _plain_cache[key]


def run_trace(folder, name, dtype, reqs, want_rough, steps, max_tokens, what, max_requests=4):
    from iian_b200.engine.replay import TraceReplayer
    want, rough = want_rough
    rp = TraceReplayer.from_folder(folder, dtype, max_tokens, BLOCK_SIZE[name], max_requests)
    got = replay_and_collect(rp, steps)
    rp.runner.check_device_status()
    rp.runner.manager.check_invariants()
    assert all(p.num_free == p.num_blocks for p in rp.runner.manager.pools), "pages were lost"
    assert len(got) == sum(len(t) for t in reqs.values())
    scale = max(w.abs().max().item() for w in want.values())
    floor = 3e-5 * max(1.0, scale) if dtype == "float32" else 3e-2 * scale
    over = []
    for (rid, pos) in sorted(got):
        assert torch.isfinite(got[(rid, pos)]).all()
        e = (got[(rid, pos)].double() - want[rid][pos]).abs().max().item()
        tol = floor + 3.0 * (rough[dtype][rid][pos] - want[rid][pos]).abs().max().item()
        assert e <= 3.0 * tol, f"{name} {dtype} {what}: first wrong logits at {(rid, pos)}: {e:.3g} > 3 x {tol:.3g}; worst {max_error(got, want)}"
        if not e <= tol:
            over.append((rid, pos, e, tol))
    # the rounded oracle is ONE draw of the rounding noise at a touchy position: a few positions may be further off than it
    assert len(over) <= 0.02 * len(got), f"{name} {dtype} {what}: {len(over)} of {len(got)} positions beyond rounding, first {over[0]}"
    return got


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_replay_under_every_cut(folders, name, dtype):
    reqs, want = requests_and_plain(folders, name, dtype)
    rounded = max(-(-len(t) // 64) * 64 for t in reqs.values())
    folder = folders[(name, dtype)]
    whole = run_trace(folder, name, dtype, reqs, want, trace_whole(reqs), rounded, "whole")
    for what, steps, cap, live in (("tail", trace_tail(reqs, 40), rounded, 4), ("portions", trace_portions(reqs), rounded, 4),
                                   ("mixed", trace_mixed(reqs, 2 * rounded, seed=1), 2 * rounded, 4),
                                   ("mixed, two live", trace_mixed(reqs, rounded + 64, seed=2, max_live=2), rounded + 64, 2)):
        got = run_trace(folder, name, dtype, reqs, want, steps, cap, what, live)
        if dtype == "float32":      # every sum has an order fixed by the token's own position: the cut changes no bit
            worst = max((got[k] - whole[k]).abs().max().item() for k in got)
            assert worst <= 2e-6, f"{name} {what}: differs from the whole prompt by {worst}"


def test_the_stream_after_every_layer(folders):
    """The float32 residual stream after each layer against the plain implementation's (what a layer still owes to the stream is
    added here by hand)."""
    from iian_b200.engine.replay import TraceReplayer
    for name in ("K", "N"):
        toks = random_tokens(CONFIGS[name]["vocab"], 21, 3)
        cfg, w = plain.load_folder(folders[(name, "float32")])
        _, streams = plain.forward(cfg, w, toks, return_layers=True)
        rp = TraceReplayer.from_folder(folders[(name, "float32")], "float32", 64, 16, 2)
        seen = []

        def spy(fn):
            def run(residual, delta, ctx, cache, writes_cache, select_rows):
                res, d = fn(residual, delta, ctx, cache, writes_cache, select_rows)
                seen.append((res.double() + owed(d)).cpu())
                return res, d
            return run
        for b in rp.model.blocks:
            b.forward = spy(b.forward)
        rp.run_step({"step": 0, "entries": [{"id": "a", "tokens": toks, "want": list(range(21))}], "end": ["a"]})
        assert len(seen) == streams.shape[0]
        for i, x in enumerate(seen):
            assert (x - streams[i]).abs().max() < 3e-5 * max(1.0, streams[i].abs().max().item()), f"{name}: layer {i}"


def test_which_kernels_serve_a_bfloat16_model(folders):
    """Heads of 128: prompts on the tcgen05 attention, decoded tokens on the fused kernel, activations inside the products."""
    from iian_b200.engine.replay import TraceReplayer
    rp = TraceReplayer.from_folder(folders[("N", "bfloat16")], "bfloat16", 256, 16, 2)
    before = launches()
    rp.run_step({"step": 0, "entries": [{"id": "a", "tokens": random_tokens(331, 150, 1), "want": [149]}], "end": []})
    ran = launched(before)
    assert ran["capped attention (tcgen05)"] == 4 and ran["head_norm_store"] == 4 and ran["gemm_tcgen05_gated"] >= 1, ran
    assert "gated_act" not in ran and "window_attention" not in ran
    before = launches()
    rp.run_step({"step": 1, "entries": [{"id": "a", "tokens": [5], "want": [0]}], "end": ["a"]})
    ran = launched(before)
    assert ran["attention_decode_fused"] == 4 and "head_norm_store" not in ran and ran["gemm_stream_gated"] >= 1 and "gated_act" not in ran, ran


def plant_a_far_question(w, asker: int, answer: int) -> None:
    """Two tokens whose rows outweigh their positions' point one way each wherever they stand; the first layer's queries see the one and
    its keys the other through the same direction of a head, so that the one asks for the other."""
    g = torch.Generator().manual_seed(7)
    width = w["embed"].shape[1]
    u = torch.sign(torch.randn(128, generator=g))
    for tok, name in ((asker, "l0.mix.q"), (answer, "l0.mix.k")):
        a = torch.randn(width, generator=g)
        a[0] = 0.0
        w["embed"][tok] = a * 0.3
        a = a / a.norm()
        w[name][:] = w[name] + 0.5 * u.repeat(w[name].shape[0] // 128)[:, None] * a[None, :]
    w["l0.norm1"][1:] = 3.0                  # what the first layer's attention says is loud in the stream
    # the answer's value is another than the mean of the rest
    w["l0.mix.v"][:] = w["l0.mix.v"] + 0.5 * torch.sign(torch.randn(128, generator=g))[:, None] * (w["embed"][answer] / w["embed"][answer].norm())[None, :]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_a_far_key(folders, dtype):
    """200 tokens decoded one by one behind a short prompt (over page and tile borders), and a token whose row is large, met once
    early and asked for again at the end."""
    reqs, want = requests_and_plain(folders, "K", dtype, [230], seed=90)
    run_trace(folders[("K", dtype)], "K", dtype, reqs, want, trace_tail(reqs, 200), 256, "long decoding")
    for name, seed in (("N", 92), ("L", 93)):          # the tensor-core kernels
        reqs, want = requests_and_plain(folders, name, dtype, [300, 270], seed=seed)
        run_trace(folders[(name, dtype)], name, dtype, reqs, want, trace_tail(reqs, 150), 320, "long decoding")
        run_trace(folders[(name, dtype)], name, dtype, reqs, want, trace_mixed(reqs, 640, seed=5), 640, "long, mixed")
    d = folders[("N", dtype)] + "_far"
    if not os.path.isdir(d):
        cfg, w = plain.load_folder(folders[("N", dtype)])
        from iian_b200.weights.safetensors_io import write_safetensors
        w = {k: (v.float() if v.is_floating_point() else v) for k, v in w.items()}
        plant_a_far_question(w, asker=9, answer=7)
        os.makedirs(d)
        write_safetensors(os.path.join(d, "model.safetensors"), {k: (v.to(torch.bfloat16) if v.is_floating_point() else v) for k, v in w.items()})
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cfg, f)
    toks = [t if t not in (7, 9) else 8 for t in random_tokens(331, 400, 3)]
    toks[4] = 7
    toks[-1] = toks[-30] = 9
    cfg, w = plain.load_folder(d)
    other = plain.forward(cfg, w, toks[:4] + [8] + toks[5:])
    reqs, want = requests_and_plain(folders, "N", dtype, folder=d, reqs={"far": toks})
    shift = (other[-1] - want[0]["far"][-1]).abs().max() / want[0]["far"].abs().max()
    assert shift > 0.08, f"the far token must matter: {shift}"
    run_trace(d, "N", dtype, reqs, want, trace_whole(reqs), 448, "far key, whole")
    run_trace(d, "N", dtype, reqs, want, trace_tail(reqs, 40), 448, "far key, decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["L", "N"])
def test_greedy_generation_through_the_entry_point(folders, name, dtype):
    from iian_b200 import EngineConfig, SchedulerConfig
    from iian_b200.engine.engine import Engine
    cfg, w = plain.load_folder(folders[(name, dtype)])
    prompts = [random_tokens(CONFIGS[name]["vocab"], n, 70 + i) for i, n in enumerate([1, 6, 30, 50, 77])]
    want = []
    for p in prompts:
        toks, margins = list(p), []
        for _ in range(10):
            row = plain.forward(cfg, w, toks)[-1]
            top = torch.topk(row, 2).values
            margins.append((top[0] - top[1]).item() / row.abs().max().item())
            toks.append(int(torch.argmax(row)))
        want.append((toks[len(p):], margins))
    for kw in (dict(budget=1024, kv_cache_tokens=1024, cuda_graphs=True), dict(budget=13, kv_cache_tokens=1024, cuda_graphs=True),
               dict(budget=64, kv_cache_tokens=128, cuda_graphs=False), dict(budget=256, kv_cache_tokens=1024, enable_prefix_caching=True)):
        sched = SchedulerConfig(max_num_batched_tokens=kw.pop("budget"), max_num_seqs=8)
        eng = Engine(folders[(name, dtype)], EngineConfig(dtype=dtype, block_size=BLOCK_SIZE[name], sched=sched, max_model_len=128, **kw))
        for _ in range(2 if kw.get("enable_prefix_caching") else 1):
            got = eng.generate(prompts, max_tokens=10, temperature=0.0)
            for g, (wt, margins) in zip(got, want):
                for k, (a, b) in enumerate(zip(g, wt)):
                    if a != b:
                        assert dtype == "bfloat16" and margins[k] < 0.05, f"{kw}: token {k}: {g} vs {wt} (margin {margins[k]:.4f})"
                        break
        if kw.get("cuda_graphs"):
            assert eng.runner.num_graphs >= 1
        eng.cache.check_invariants()
        if not kw.get("enable_prefix_caching"):
            assert all(p.num_free == p.num_blocks for p in eng.cache.pools)


def test_trace_runner_as_a_program(folders, tmp_path):
    reqs, (want, _) = requests_and_plain(folders, "M", "float32")
    steps = trace_mixed(reqs, 384, seed=4)
    out = tmp_path / "out"
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folders[("M", "float32")], "--dtype", "float32",
                           "--out", str(out), "--max-tokens", "384", "--block-size", "32"],
                          input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    fed = {}
    for s in steps:
        rows = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, 97)
        r = 0
        for ent in s["entries"]:
            for k in ent["want"]:
                p = fed.get(ent["id"], 0) + k
                assert np.abs(rows[r] - want[ent["id"]][p].numpy()).max() < 1e-4
                r += 1
            fed[ent["id"]] = fed.get(ent["id"], 0) + len(ent["tokens"])

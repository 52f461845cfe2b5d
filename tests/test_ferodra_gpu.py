"""Ferodra on the GPU.  Each new kernel alone against the plain functions of tests/plain_ferodra.py (the norm by tanh with a
normalised addend and a vector for every row; interleaved rotation and the cache write; the difference of two softmax maps with a
stand-out key for either map far back, at page and tile borders and at the query itself, as rows of a portion and as decoded
tokens, with scores far inside and far beyond the cap, through the general kernel, the mma.sync kernel with its cluster merge and
the tcgen05 kernel; the delta rule with one decay per head in every lane form, cut into steps, with slots used again; the router
with its correction, identity outputs and the gated shared expert); then whole models under every way of cutting the work, in
32-bit and in bfloat16; greedy generation through the engine's entry point with and without CUDA graphs; the trace runner as a
program."""
import json
import math
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from helpers import max_error, random_tokens, replay_and_collect, trace_mixed, trace_portions, trace_tail, trace_whole
import plain_ferodra as plain
from ferodra_cases import BLOCK_SIZE, CONFIGS, owed, plain_logits, rounded_plain, write_case

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


def K():
    from iian_b200 import ops
    return ops.kernels()


def close(got, want, dtype, what, rel16=2e-2, abs32=2e-5):
    got, want = got.double().cpu(), want.double().cpu()
    tol = abs32 * max(1.0, want.abs().max().item()) if dtype == "float32" else rel16 * want.abs().max().item()
    err = (got - want).abs().max().item()
    assert err <= tol, f"{what} [{dtype}]: max error {err:.3g} > {tol:.3g}"


# ---- row-wise kernels ---------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n, h", [(5, 72), (3, 100), (4, 1000), (2, 4100), (3, 30), (700, 128), (3000, 260)])
def test_norm_by_tanh_with_a_normalised_addend(dtype, n, h):
    g = torch.Generator().manual_seed(h)
    x = torch.randn(n, h, generator=g) * 3
    y = (torch.randn(n, h, generator=g) * 7).to(DT[dtype])
    u, c, w, b, row = (torch.randn(h, generator=g) for _ in range(5))
    W = {"u": u.double(), "u.alpha": torch.tensor(0.3, dtype=F64), "u.b": c.double(), "w": w.double(), "w.alpha": torch.tensor(0.7, dtype=F64), "w.b": b.double()}
    for with_y, with_u, with_row, with_out in ((1, 1, 0, 1), (1, 1, 1, 1), (1, 0, 0, 1), (0, 0, 0, 1), (0, 0, 1, 0), (1, 1, 0, 0)):
        res = x.to(DEV).clone()
        out = torch.empty(n, h, device=DEV, dtype=DT[dtype]) if with_out else None
        K().tanh_add_tanh(res, y.to(DEV) if with_y else None, 0.3, u.to(DEV) if with_u else None, c.to(DEV) if with_u else None,
                          row.to(DEV) if with_row else None, 0.7, w.to(DEV) if with_out else None, b.to(DEV) if with_out else None, out)
        s = x.double()
        if with_y:
            s = s + (plain.tanh_norm(y.double(), W, "u") if with_u else y.double())
        if with_row:
            s = s + row.double()
        close(res, s, "float32", f"the stream, width {h}")
        if with_out:
            close(out, plain.tanh_norm(s, W, "w"), dtype, f"the next norm, width {h}", rel16=8e-3)
    res = x.to(DEV).clone()
    K().add_row(res, row.to(DEV))
    close(res, x.double() + row.double(), "float32", "a vector for every row", abs32=1e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_squared_positive_part(dtype):
    for n in (7, 64, 4096 * 3 + 4):
        x = (torch.randn(n, generator=torch.Generator().manual_seed(n)) * 3).to(DT[dtype])
        out = torch.empty(n, dtype=DT[dtype], device=DEV)
        K().relu2(x.to(DEV), out)
        close(out, torch.relu(x.double()) ** 2, dtype, "squared positive part", rel16=5e-3)


# ---- rotation and cache write ------------------------------------------------------------------------------
def _fill_cache(dtype, H, G, d, dv, freqs, magnitude, positions, page, seed):
    """Projections of len(positions) tokens of one sequence through the kernels into a paged cache of scattered pages; returns
    what the plain functions make of the same rows."""
    g = torch.Generator().manual_seed(seed)
    n = len(positions)
    nq, nk, nv = H * 2 * d, G * 2 * d, G * dv
    proj = torch.randn(n, nq + nk + nv + 8, generator=g).to(DT[dtype])            # the mixer's columns start behind 8 others
    n_used = -(-(max(positions) + 1) // page)
    order = torch.randperm(n_used + 3, generator=g)[:n_used].to(torch.int32)
    kc = torch.zeros(n_used + 3, G, page, 2 * d, dtype=DT[dtype], device=DEV)
    vc = torch.zeros(n_used + 3, G, page, dv, dtype=DT[dtype], device=DEV)
    pos = torch.tensor(positions, dtype=torch.int32)
    slots = (order[(pos // page).long()] * page + pos % page).to(torch.int32)
    q = torch.empty(n, nq, dtype=DT[dtype], device=DEV)
    rot = 2 * freqs.numel()
    table = None
    if rot:
        table = torch.empty(n, rot // 2, 2, device=DEV)
        K().rotary_table_scaled(freqs.to(DEV), pos.to(DEV), rot // 2, magnitude, table)
    K().rotate_pairs_store(proj.to(DEV)[:, 8:], 0, nq, nq + nk, q, kc, vc, table, slots.to(DEV), num_heads=2 * H, num_kv_heads=G, maps=2,
                           k_dim=d, v_dim=dv, rot_dim=rot)
    p = proj.double()[:, 8:]
    qw = plain.rotate_neighbours(p[:, :nq].reshape(n, 2 * H, d), pos, freqs, magnitude).view(n, H, 2, d)
    kw = plain.rotate_neighbours(p[:, nq:nq + nk].reshape(n, 2 * G, d), pos, freqs, magnitude).view(n, G, 2, d)
    return SimpleNamespace(q=q, kc=kc, vc=vc, order=order, slots=slots, pos=pos, q_want=qw, k_want=kw, v_want=p[:, nq + nk:].reshape(n, G, dv))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, d, dv, rot", [(6, 2, 16, 24, 8), (3, 3, 40, 24, 40), (2, 1, 64, 128, 0), (4, 2, 64, 128, 20), (1, 1, 22, 7, 10),
                                              (5, 1, 200, 8, 100)])
def test_rotation_of_neighbours_and_cache_write(dtype, H, G, d, dv, rot):
    positions = [0, 1, 7, 8, 9, 70000][: 6 if rot else 5]                     # a far position: the angle is a float64 product
    freqs, mag = plain.rotation({"dims": rot, "base": 777.0, "scaling": {"factor": 4.0, "original": 40, "fast": 16.0, "slow": 1.0}} if rot else None)
    c = _fill_cache(dtype, H, G, d, dv, freqs, mag, positions, 8, seed=d)
    close(c.q.view(-1, H, 2, d), c.q_want, dtype, "rotated queries", rel16=1e-2)
    cells = c.slots.long().to(DEV)
    close(c.kc.permute(0, 2, 1, 3).reshape(-1, G, 2, d)[cells], c.k_want, dtype, "keys in their cells", rel16=1e-2)
    assert torch.equal(c.vc.permute(0, 2, 1, 3).reshape(-1, G, dv)[cells].cpu().double(), c.v_want), "values go in exactly as projected"
    assert int((c.kc != 0).any(-1).any(1).sum()) == len(positions), "cells of other tokens were written"
    # a padding token (cell -1) stores nothing
    before = c.kc.clone()
    proj = torch.randn(1, H * 2 * d + G * (2 * d + dv), device=DEV).to(DT[dtype])
    table = torch.ones(1, rot // 2, 2, device=DEV) if rot else None
    K().rotate_pairs_store(proj, 0, H * 2 * d, (H + G) * 2 * d, torch.empty(1, H * 2 * d, device=DEV, dtype=DT[dtype]), c.kc, c.vc, table,
                           torch.tensor([-1], dtype=torch.int32, device=DEV), num_heads=2 * H, num_kv_heads=G, maps=2, k_dim=d, v_dim=dv,
                           rot_dim=rot)
    assert torch.equal(before, c.kc)


def test_the_positions_table_follows_the_plug_ins_frequencies():
    from iian_b200.config.spec import PartSpec
    from iian_b200.parts.position import Rotary, ScaledRotary
    for rot in ({"dims": 48, "base": 1e6, "scaling": {"factor": 4.0, "original": 512, "fast": 32.0, "slow": 1.0}},
                {"dims": 20, "base": 300.0, "scaling": {"factor": 2.0, "original": 64, "fast": 2.0, "slow": 2.0}}, {"dims": 16, "base": 100.0}):
        params = {"dim": rot["dims"], "base": rot["base"], "style": "interleaved"}
        part = ScaledRotary(PartSpec("scaled_rotary", dict(params, scaling=dict(rot["scaling"], kind="ramp"))), torch.float32, DEV) if "scaling" in rot \
            else Rotary(PartSpec("rotary", params), torch.float32, DEV)
        f, m = plain.rotation(rot)
        assert (part.inv_freq64.cpu() - f).abs().max() < 1e-15 and part.magnitude == pytest.approx(m)


# ---- attention ---------------------------------------------------------------------------------------------
ATTENTION = [  # H, G, d, dv, page, n, cap
    (6, 2, 16, 24, 16, 300, 4.0), (4, 4, 64, 128, 8, 300, 20.0), (8, 2, 64, 128, 16, 700, 25.0), (3, 1, 24, 8, 16, 150, None), (4, 1, 64, 128, 32, 1500, None),
    (4, 2, 64, 128, 16, 2600, 10.0), (2, 2, 40, 200, 16, 260, 15.0), (5, 1, 22, 12, 8, 90, 6.0), (32, 1, 64, 128, 64, 400, 30.0), (6, 3, 64, 128, 24, 200, 12.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, d, dv, page, n, cap", ATTENTION)
def test_difference_of_two_maps(dtype, H, G, d, dv, page, n, cap):
    """Keys are made to stand out by putting a multiple of a query's map into their cells: a far one for map 1 only, a far one for
    map 2 only, one at a page's and a tile's last and first place, the query's own position.  Queries: a portion of the last 7
    tokens, the same one by one, the first ones, long portions.  Maps of 64 over values of 128 run on the tensor-core kernels in
    bfloat16."""
    freqs, mag = plain.rotation({"dims": min(d, 16) // 2 * 2, "base": 777.0})
    c = _fill_cache(dtype, H, G, d, dv, freqs, mag, list(range(n)), page, seed=H * d)
    first = torch.arange(G) * (H // G)
    cut = 64 if n > 80 else 32
    marks = [(1, n - 1, 0), (2, n - 2, 1), (cut - 1, n - 3, 0), (cut, n - 4, 0), (page - 1, n - 5, 1), (page, n - 6, 1), (n - 7, n - 7, 0)]
    for j, asker, m in marks:
        key = (1.5 * c.q_want[asker, first, m]).to(DT[dtype])                              # [G, d], for one map only
        cell = int(c.slots[j])
        c.kc[cell // page, :, cell % page, m * d:(m + 1) * d] = key.to(DEV)
        c.k_want[j, :, m] = key.double()
    scale, lam, diff, eps = (5.0 if n < 2000 else 7.0) / d, 0.4, 0.3, 1e-5
    want = plain.map_difference(c.q_want, c.k_want, c.v_want, scale, cap, lam, diff, eps).reshape(n, H * dv)
    for j, asker, m in marks:                                                              # without its stand-out key a row is another
        g = torch.softmax((c.q_want[asker, 0, m] @ c.k_want[: asker + 1, 0, m].T) * scale, -1)
        assert g[j] > 0.1, "the stand-out key must matter"
    if cap:
        uncapped = plain.map_difference(c.q_want[n - 9:], c.k_want, c.v_want, scale, None, lam, diff, eps, n - 9).reshape(9, H * dv)
        assert (uncapped - want[n - 9:]).abs().max() > 5e-3, "the cap must show"
    bt = torch.full((1, max(64, c.order.numel())), -1, dtype=torch.int32)
    bt[0, : c.order.numel()] = c.order
    from iian_b200.ops import cuda_backend
    before = dict(cuda_backend.LAUNCHES_BY_ENTRY)
    for rows in (list(range(n - 7, n)), [n - 4], [n - 3], [n - 2], [n - 1], [0], list(range(0, 3)), list(range(max(0, n - 200), n)),
                 list(range(0, min(n, 130))), list(range(cut - 1, cut + 2))):
        r = torch.tensor(rows)
        meta = SimpleNamespace(positions=c.pos[r].to(DEV), seq_of_token=torch.zeros(len(rows), dtype=torch.int32, device=DEV),
                               cu_q=torch.tensor([0, len(rows)], dtype=torch.int32, device=DEV),
                               ctx_len=torch.tensor([rows[-1] + 1], dtype=torch.int32, device=DEV), block_table=bt.to(DEV),
                               num_seqs=1, num_tokens=len(rows), max_q_len=len(rows), max_ctx=rows[-1] + 1)
        for split in ((None, 1, 2, 4, 8, 16) if len(rows) == 1 else (None,)):
            out = torch.empty(len(rows), H * dv, dtype=DT[dtype], device=DEV)
            K().difference_attention(c.q[r.to(DEV)], c.kc, c.vc, out, meta, num_heads=H, num_kv_heads=G, k_dim=d, v_dim=dv, scale=scale,
                                     softcap=cap, lam=lam, factor=1.0 - diff, eps=eps, n_split=split)
            close(out, want[r], dtype, f"attention rows {rows[0]}..{rows[-1]}, parts {split}", rel16=2.5e-2)
    K().check_device_status()
    fast = dtype == "bfloat16" and d == 64 and dv == 128
    ran = {k: v - before.get(k, 0) for k, v in cuda_backend.LAUNCHES_BY_ENTRY.items() if v != before.get(k, 0)}
    assert ("difference_attention" not in ran) == fast, f"which kernel served it: {ran}"
    if fast:
        assert "difference_attention_mma" in ran and ("attention_tc_difference" in ran) == (page in (8, 16, 32, 64, 128)), ran


@pytest.mark.parametrize("G, rep, lengths", [(2, 3, [1, 70, 500, 33, 64, 65]), (8, 4, [900, 2, 128, 1]), (1, 16, [300] * 40)])
def test_difference_attention_batches(G, rep, lengths):
    """Several sequences in one launch (decoded tokens beside portions, a padding sequence, many sequences: the TMA form), scores
    small enough for the polynomial and others beyond the cap."""
    H, d, dv, page = G * rep, 64, 128, 16
    for strength, cap in ((0.02, 30.0), (0.6, 9.0)):
        for tail in (1, 5, 40):
            g = torch.Generator().manual_seed(tail)
            S = len(lengths)
            n_pages = sum(-(-n // page) for n in lengths)
            order = torch.randperm(n_pages, generator=g).to(torch.int32)
            kc = torch.randn(n_pages, G, page, 2 * d, generator=g).to(torch.bfloat16)
            vc = torch.randn(n_pages, G, page, dv, generator=g).to(torch.bfloat16)
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
            q = torch.randn(cu[-1], H * 2 * d, generator=g).to(torch.bfloat16)
            i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
            meta = SimpleNamespace(positions=i32(pos), seq_of_token=i32(seq), cu_q=i32(cu), ctx_len=i32(lengths + [1]), block_table=bt.to(DEV),
                                   num_seqs=S + 1, num_tokens=cu[-1], max_q_len=min(tail, max(lengths)), max_ctx=max(lengths))
            out = torch.empty(cu[-1], H * dv, dtype=torch.bfloat16, device=DEV)
            K().difference_attention(q.to(DEV), kc.to(DEV), vc.to(DEV), out, meta, num_heads=H, num_kv_heads=G, k_dim=d, v_dim=dv, scale=strength,
                                     softcap=cap, lam=0.5, factor=0.6, eps=1e-6)
            K().check_device_status()
            for s, n in enumerate(lengths[:6]):
                js = torch.arange(n)
                cells = bt[s, js // page].long(), js % page
                kk = kc.double()[cells[0], :, cells[1]].view(n, G, 2, d)
                vv = vc.double()[cells[0], :, cells[1]]
                a, b = cu[s], cu[s + 1]
                want = plain.map_difference(q.double()[a:b].view(b - a, H, 2, d), kk, vv, strength, cap, 0.5, 0.4, 1e-6, n - (b - a))
                close(out[a:b], want.reshape(b - a, H * dv), "bfloat16", f"sequence {s} of {n} keys, {b - a} rows", rel16=2.5e-2)


# ---- the delta rule with one decay per head ---------------------------------------------------------------------
def _plain_delta(proj, ab, H, G, d, dv, taps, a_log, dt_bias, state=None, before=None):
    n = proj.shape[0]
    x = plain.silu(plain.short_convolution(proj, taps, before))
    q, k, v = x[:, : G * d].view(n, G, d), x[:, G * d: 2 * G * d].view(n, G, d), x[:, 2 * G * d:].view(n, H, dv)
    q, k = plain.unit_length(q) * d ** -0.5, plain.unit_length(k)
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    g = torch.exp(-torch.exp(a_log) * torch.nn.functional.softplus(ab[:, :H] + dt_bias))
    o, S = plain.delta_scan(q, k, v, torch.sigmoid(ab[:, H:]), g, state)
    return o.reshape(n, H * dv), S


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H, G, d, dv, taps", [(6, 2, 24, 40, 4), (2, 2, 16, 24, 1), (4, 1, 32, 32, 2), (1, 1, 160, 16, 4), (1, 1, 8, 8, 8), (4, 2, 64, 128, 4),
                                               (1, 1, 300, 6, 3), (5, 5, 128, 48, 4), (3, 1, 50, 20, 5), (2, 1, 512, 20, 4), (4, 2, 128, 128, 4)])
def test_delta_rule_cut_into_steps_with_slots_used_again(dtype, H, G, d, dv, taps):
    """Three sequences of unequal length walked in steps of 1 to 29 tokens beside each other and a padding sequence, against the
    plain recurrence over whole sequences; then a long sequence in one step, in a slot that was used (zeroed as at admission)."""
    g = torch.Generator().manual_seed(H * d + dv)
    lengths = [37, 5, 64, 700]
    C = 2 * G * d + H * dv
    projs = [(torch.randn(n, C + 8, generator=g) * 0.7).to(DT[dtype]) for n in lengths]
    abs_ = [torch.randn(n, 2 * H, generator=g) * 2 for n in lengths]
    conv = torch.randn(C, taps, generator=g) * 0.6
    a_log, dt_bias = torch.randn(H, generator=g) * 0.5 - 1.0, torch.randn(H, generator=g)
    want = [_plain_delta(p.double()[:, 8:], ab.double(), H, G, d, dv, conv.double(), a_log.double(), dt_bias.double())[0]
            for p, ab in zip(projs, abs_)]
    from iian_b200.engine.runner import StepContext, Workspace
    from iian_b200.parts.delta_rule import state_floats
    state = torch.zeros(4, state_floats(H, G, d, dv, taps), device=DEV)
    conv_d, a_d, dt_d = conv.to(DEV), a_log.to(DEV), dt_bias.to(DEV)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)

    def run(parts, slots):
        cu = [0]
        for p, _ in parts:
            cu.append(cu[-1] + p.shape[0])
        proj = torch.cat([p for p, _ in parts]).to(DEV)
        ab = torch.cat([a for _, a in parts]).to(DEV)
        ctx = StepContext(Workspace(torch.device(DEV)))
        ctx.cu_q, ctx.state_slots = i32(cu), i32(slots)
        ctx.seq_of_token = i32([(s if slots[s] >= 0 else -1) for s, (p, _) in enumerate(parts) for _ in range(p.shape[0])])
        ctx.max_q_len = max(p.shape[0] for p, _ in parts)
        out = torch.full((proj.shape[0], H * dv), 7.0, device=DEV)
        K().delta_rule(proj[:, 8:], 0, 0, ab[:, :H], conv_d, a_d, dt_d, state, ctx, out, num_heads=H, num_kv_heads=G, dim=d, v_dim=dv,
                       b_pre=ab[:, H:])
        return [out[cu[i]:cu[i + 1]].cpu() for i in range(len(parts))]

    slots, fed, step = [2, 0, 3], [0, 0, 0], 0
    got = [torch.zeros(n, H * dv) for n in lengths[:3]]
    sizes = [1, 7, 2, 29, 1, 1, 16, 3, 17, 2]
    while any(f < n for f, n in zip(fed, lengths)):
        take = []
        for i in range(3):
            c = min(sizes[(step + i) % len(sizes)], lengths[i] - fed[i])
            if c > 0 and (step + i) % 4 != 3:
                take.append((i, fed[i], c))
        step += 1
        if not take:
            continue
        outs = run([(projs[i][a:a + c], abs_[i][a:a + c]) for i, a, c in take] + [(projs[0][:1], abs_[0][:1])], [slots[i] for i, _, _ in take] + [-1])
        assert (outs[-1] == 0).all()
        for (i, a, c), o in zip(take, outs):
            got[i][a:a + c] = o
            fed[i] += c
    for i in range(3):
        close(got[i], want[i], "float32", f"sequence {i} of {H} heads {d} x {dv}", abs32=5e-5)
    assert (state[1] == 0).all(), "a slot no sequence had was written"
    state[2].zero_()
    close(run([(projs[3], abs_[3])], [2])[0], want[3], "float32", "a long sequence in a slot that was used before", abs32=5e-5)


# ---- experts: corrected choice, identity outputs, a gated shared expert -----------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n, experts, identity, top, width, ff, shared", [
    (1, 3, 1, 1, 64, 32, 16), (9, 5, 0, 2, 96, 48, 0), (300, 8, 4, 3, 128, 64, 96), (40, 2, 2, 4, 100, 36, 20), (17, 30, 9, 4, 64, 24, 40),
    (5, 1, 5, 2, 72, 40, 8), (600, 12, 3, 2, 256, 128, 64)])
def test_corrected_router_identity_outputs_and_the_shared_expert(dtype, n, experts, identity, top, width, ff, shared):
    from iian_b200.config.spec import PartSpec
    from iian_b200.engine.runner import StepContext, Workspace
    from iian_b200.parts.experts import RoutedExperts
    g = torch.Generator().manual_seed(n + experts)
    part = RoutedExperts(PartSpec("routed_experts", {"hidden_size": width, "num_experts": experts, "identity_experts": identity, "top": top,
                                                     "intermediate_size": ff, "activation": "relu2", "score": "softmax", "weight_scale": 1.7,
                                                     "weight_on": "output", "shared_intermediate_size": shared, "shared_gate": True}),
                         DT[dtype], torch.device(DEV))
    std = {"router": 0.2, "correction": 0.2, "shared.sg": 0.2}
    tensors = {name: (torch.randn(*ts.shape, generator=g) * std.get(name, 0.15)).to(DT[dtype]) for name, ts in part.tensors().items()}
    part.bind({k: v.to(DEV) for k, v in tensors.items()})
    h = torch.randn(n, width, generator=g).to(DT[dtype])
    out = part.forward(h.to(DEV), StepContext(Workspace(torch.device(DEV))))
    K().check_device_status()
    w64 = {k: v.double() for k, v in tensors.items()}
    cfg = {"router": {"experts": experts, "identity": identity, "top": top, "scale": 1.7}, "shared": {"ff": shared} if shared else None}
    plain.router_margins = []
    try:
        want = plain.experts_feed_forward(cfg, w64, "", h.double())
        margins = plain.router_margins[0]
    finally:
        plain.router_margins = None
    ids, _ = plain.router_choice(h.double(), w64, "", top, 1.7)
    safe = margins > (1e-6 if dtype == "float32" else 4e-3)            # rows where rounding cannot change the choice
    assert safe.sum() > 0.6 * n
    if identity and n > 8:
        assert (ids >= experts).any() and (ids < experts).any()
    close(out[safe.to(DEV)], want[safe], dtype, "experts' weighted sum, identity outputs, shared expert", rel16=3e-2, abs32=3e-5)


# ---- whole models --------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("ferodra_gpu")
    out = {(name, "float32"): write_case(root, name) for name in CONFIGS}
    out.update({(name, "bfloat16"): write_case(root, name, router_step=2.0) for name in CONFIGS})     # see spread_corrections
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
                                   ("mixed, two slots", trace_mixed(reqs, rounded + 64, seed=2, max_live=2), rounded + 64, 2)):
        got = run_trace(folder, name, dtype, reqs, want, steps, cap, what, live)
        if dtype == "float32":      # every sum has an order fixed by the token's own position: the cut changes no bit
            worst = max((got[k] - whole[k]).abs().max().item() for k in got)
            assert worst <= 2e-6, f"{name} {what}: differs from the whole prompt by {worst}"


def test_the_stream_after_every_layer_run(folders):
    """The float32 residual stream after each layer run against the plain implementation's (what a layer still owes to the
    stream is added here by hand)."""
    from iian_b200.engine.replay import TraceReplayer
    for name, vocab in (("K", 211), ("N", 331)):
        toks = random_tokens(vocab, 21, 3)
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
            assert (x - streams[i]).abs().max() < 3e-5 * max(1.0, streams[i].abs().max().item()), f"{name}: layer run {i}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_a_far_key(folders, dtype):
    """200 tokens decoded one by one behind a short prompt (over page and tile borders, the recurrences run on), and a token whose
    embedding is large, met once early and again at the end."""
    reqs, want = requests_and_plain(folders, "K", dtype, [230], seed=90)
    run_trace(folders[("K", dtype)], "K", dtype, reqs, want, trace_tail(reqs, 200), 256, "long decoding")
    for name, seed in (("N", 92), ("L", 93)):          # maps of 64 over values of 128: the tensor-core kernels
        reqs, want = requests_and_plain(folders, name, dtype, [300, 270], seed=seed)
        run_trace(folders[(name, dtype)], name, dtype, reqs, want, trace_tail(reqs, 150), 320, "long decoding")
        run_trace(folders[(name, dtype)], name, dtype, reqs, want, trace_mixed(reqs, 640, seed=5), 640, "long, mixed")
    d = folders[("N", dtype)] + "_far"
    if not os.path.isdir(d):
        cfg, w = plain.load_folder(folders[("N", dtype)])
        from iian_b200.weights.safetensors_io import write_safetensors
        w = {k: (v.float() if v.is_floating_point() else v) for k, v in w.items()}
        w["embed"][7] *= 6.0
        os.makedirs(d)
        write_safetensors(os.path.join(d, "model.safetensors"), {k: (v.to(torch.bfloat16) if v.is_floating_point() else v) for k, v in w.items()})
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cfg, f)
    toks = [t if t != 7 else 8 for t in random_tokens(331, 400, 3)]
    toks[4] = toks[-1] = toks[-30] = 7
    reqs, want = requests_and_plain(folders, "N", dtype, folder=d, reqs={"far": toks})
    run_trace(d, "N", dtype, reqs, want, trace_whole(reqs), 448, "far key, whole")
    run_trace(d, "N", dtype, reqs, want, trace_tail(reqs, 40), 448, "far key, decoded")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(folders, dtype):
    from iian_b200 import EngineConfig, SchedulerConfig
    from iian_b200.engine.engine import Engine
    name = "L"
    cfg, w = plain.load_folder(folders[(name, dtype)])
    prompts = [random_tokens(300, n, 70 + i) for i, n in enumerate([1, 6, 30, 50, 77])]
    want = []
    for p in prompts:
        toks, margins = list(p), []
        for _ in range(10):
            row = plain.forward(cfg, w, toks)[-1]
            top = torch.topk(row, 2).values
            margins.append((top[0] - top[1]).item())
            toks.append(int(torch.argmax(row)))
        want.append((toks[len(p):], margins))
    for kw in (dict(budget=1024, kv_cache_tokens=1024, cuda_graphs=True), dict(budget=13, kv_cache_tokens=1024, cuda_graphs=True),
               dict(budget=64, kv_cache_tokens=128, cuda_graphs=False)):
        sched = SchedulerConfig(max_num_batched_tokens=kw.pop("budget"), max_num_seqs=8)
        eng = Engine(folders[(name, dtype)], EngineConfig(dtype=dtype, block_size=BLOCK_SIZE[name], sched=sched, max_model_len=128, **kw))
        got = eng.generate(prompts, max_tokens=10, temperature=0.0)
        for g, (wt, margins) in zip(got, want):
            for k, (a, b) in enumerate(zip(g, wt)):
                if a != b:
                    assert dtype == "bfloat16" and margins[k] < 0.05, f"{kw}: token {k}: {g} vs {wt} (margin {margins[k]:.4f})"
                    break
        if kw.get("cuda_graphs"):
            assert eng.runner.num_graphs >= 1
        eng.cache.check_invariants()
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

"""Ruvalix on the GPU: every new kernel against its plain reference at sizes of its own, then
bin/trace_run replaying requests whole, decoded token by token, in portions and mixed with pages and
slots used again, in 32-bit and bfloat16, against the plain model; keys just inside and just outside a window
and far back; greedy generation through ``Engine.generate`` (graphs, steps launched ahead) and the command
line; configurations drawn at random."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import helpers
from tests.gpu_helpers import STORE, _Ctx, batches, close, rnd, step_batch, up64
from tests.helpers import TraceRunner
from tests.plain import ruvalix_plain as rp
from tests.ruvalix_cases import CASES, edge_model, model_dir, plain_logits, random_tokens, weights, write

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", params=["float32", "bfloat16"])
def both(request):
    from garuda_b200.kernels.ops import CudaOps
    from tests.plain.cpu_ops import CpuOps
    dt = STORE[request.param]
    return CudaOps("cuda:0", tensor_cores=dt == torch.bfloat16), CpuOps(), dt


# ---------------------------------------------------------------------------- kernels
@pytest.mark.parametrize("T,d", [(1, 44), (37, 200), (5, 1030), (3, 4096), (700, 15), (300, 2048), (2, 10244), (301, 9000)])
def test_norms_around_a_residual(both, T, d):
    """The output's norm, the sum, a row, and the next norm or a rounded copy, each with and without the others;
    destinations that are columns of a wider row."""
    ops, ref, dt = both
    x, y, w, row, w2 = rnd(T, d, scale=3.0, seed=1), rnd(T, d, scale=0.2, seed=2), rnd(d, seed=3), rnd(d, seed=4), rnd(d, seed=5)
    tol = 1e-2 if dt == torch.bfloat16 else 3e-6
    for use in ((1, 1, 0, 1), (1, 1, 1, 1), (1, 0, 0, 0), (0, 0, 1, 1), (0, 0, 0, 1), (1, 1, 0, 2), (0, 0, 0, 2), (1, 1, 0, 3)):
        kw = dict(y=y if use[0] else None, weight=w if use[1] else None, eps=1e-5, row=row if use[2] else None,
                  then_weight=w2 if use[3] in (1, 3) else None, then_eps=1e-4)
        wide = 2 * d if use[3] >= 2 else d
        want, got = torch.zeros(T, wide, dtype=dt), torch.zeros(T, wide, dtype=dt, device="cuda")
        xr, xg = x.clone(), x.clone().cuda()
        ref.residual_norm(xr, out=want[:, wide - d:] if use[3] else None, **kw)
        ops.residual_norm(xg, out=got[:, wide - d:] if use[3] else None, **{k: v.cuda() if torch.is_tensor(v) else v for k, v in kw.items()})
        close(xg, xr, torch.float32, f"residual {use}", 3e-6)
        close(got, want, dt, f"out {use}", tol)
        assert not got[:, :wide - d].any()


@pytest.mark.parametrize("T,d", [(1, 44), (70, 200), (5, 1030)])
def test_normed_embedding(both, T, d):
    ops, ref, dt = both
    table, w = rnd(50, d, dtype=dt, scale=0.1, seed=1), rnd(d, seed=2)
    ids = torch.randint(0, 50, (T,), dtype=torch.int32, generator=torch.Generator().manual_seed(3))
    for paired in (True, False):
        xr, xg = torch.empty(T, d), torch.empty(T, d, device="cuda")
        pr, pg = (torch.empty(T, 2 * d, dtype=dt), torch.empty(T, 2 * d, dtype=dt, device="cuda")) if paired else (None, None)
        ref.embedding_norm(table, ids, w, 1e-5, xr, pr)
        ops.embedding_norm(table.cuda(), ids.cuda(), w.cuda(), 1e-5, xg, pg)
        close(xg, xr, torch.float32, "embedding", 3e-6)
        if paired:
            close(pg, pr, dt, "pair", 1e-2 if dt == torch.bfloat16 else 3e-6)


@pytest.mark.parametrize("T,E,K,top,groups", [(1, 6, 44, 3, (3, 2)), (9, 16, 128, 2, (2, 1)), (150, 12, 192, 4, None), (33, 64, 256, 8, (8, 3)),
                                              (5, 40, 64, 1, (40, 1)), (7, 12, 64, 12, (4, 4)), (3, 300, 64, 32, (50, 20))])
@pytest.mark.parametrize("score", ["softmax_all", "sigmoid"])
def test_choice_by_corrected_scores_in_groups(both, T, E, K, top, groups, score):
    """Corrections that turn the choice around, choice scores that are all negative, every group and one of them."""
    ops, ref, dt = both
    h, w = rnd(T, K, dtype=dt, seed=1), rnd(E, K, dtype=dt, scale=0.3, seed=2)
    for shift in (0.0, -3.0):
        corr = rnd(E, scale=0.2, seed=3) + shift
        i1, i2 = torch.empty(T, top, dtype=torch.int32), torch.empty(T, top, dtype=torch.int32, device="cuda")
        w1, w2 = torch.empty(T, top), torch.empty(T, top, device="cuda")
        ref.route_topk(h, w, None, top, i1, w1, score=score, correction=corr, groups=groups)
        ops.route_topk(h.cuda(), w.cuda(), None, top, i2, w2, score=score, correction=corr.cuda(), groups=groups)
        same = (i1 == i2.cpu()).all(-1)
        assert same.float().mean() >= 0.97          # (a row of many near-equal scores may fall the other way)
        close(w2.cpu()[same], w1[same], torch.float32, "weights", 1e-5)
        assert (w2 > 0).all()


@pytest.mark.parametrize("T,E,identity,K,F,top,shared_scale", [(1, 5, 1, 44, 24, 3, 1.0), (9, 4, 4, 128, 64, 4, 0.5), (150, 6, 2, 192, 72, 2, 1.0),
                                                              (700, 8, 4, 256, 128, 3, 1.0), (65, 3, 1, 64, 200, 1, 1.0)])
def test_experts_that_return_their_input(both, T, E, identity, K, F, top, shared_scale):
    """Few pairs, many pairs and the plain kernel; tokens whose experts are all of that kind."""
    ops, ref, dt = both
    h = rnd(T, K, dtype=dt, seed=1)
    gates, ups = [rnd(F, K, dtype=dt, scale=0.2, seed=10 + e) for e in range(E)], [rnd(F, K, dtype=dt, scale=0.2, seed=40 + e) for e in range(E)]
    down = rnd(E, K, F, dtype=dt, scale=0.2, seed=3)
    g = torch.Generator().manual_seed(4)
    ids = torch.stack([torch.randperm(E + identity, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    if identity >= top:
        ids[T // 2] = torch.arange(E, E + top)
    wts, x = torch.rand(T, top, generator=g), rnd(T, K, seed=5)
    for on in (True, False):
        want, got = x.clone(), x.clone().cuda()
        ref.routed_feed_forward(_Ctx("cpu"), h, ref.pack_expert_gate_up(gates, ups), down, ids, wts, want, "silu", 0.0, shared_scale, identity=on)
        ops.routed_feed_forward(_Ctx(), h.cuda(), ops.pack_expert_gate_up([t.cuda() for t in gates], [t.cuda() for t in ups]), down.cuda(), ids.cuda(),
                                wts.cuda(), got, "silu", 0.0, shared_scale, identity=on)
        close(got, want, dt, f"experts, identity {on}")


@pytest.mark.parametrize("T", [1, 9, 150, 700])
def test_experts_rows_are_added_up_by_the_pass_behind_them(T):
    """Few pairs and many, with and without a base and experts that return their input: the pass over the residual behind
    them gives what it gives behind their sum; sizes of the plain kernels leave no rows."""
    from garuda_b200.kernels.ops import CudaOps
    ops, bf = CudaOps("cuda:0"), torch.bfloat16
    for E, identity, K, F, top, leaves in ((6, 3, 128, 64, 3, True), (5, 0, 1032, 40, 2, True), (6, 3, 44, 24, 3, False)):
        h, down = rnd(T, K, dtype=bf, seed=1).cuda(), rnd(E, K, F, dtype=bf, scale=0.3, seed=2).cuda()
        gu = ops.pack_expert_gate_up([rnd(F, K, dtype=bf, scale=0.2, seed=9 + e).cuda() for e in range(E)], [rnd(F, K, dtype=bf, scale=0.2, seed=40 + e).cuda() for e in range(E)])
        ids = torch.stack([torch.randperm(E + identity)[:top] for _ in range(T)]).to(torch.int32).cuda()
        wts, base, x = torch.rand(T, top).cuda(), rnd(T, K, seed=3).cuda(), rnd(T, K, seed=4).cuda()
        w, w2 = rnd(K, seed=5).cuda(), rnd(K, seed=6).cuda()
        for b in (base, None):
            rows = ops.expert_rows(_Ctx(), h, gu, down, ids, wts, "silu", 0.0, identity=identity > 0, base=b)
            assert (rows is not None) == leaves
            if not leaves:
                continue
            y = b.clone() if b is not None else torch.zeros(T, K, device="cuda")
            ops.routed_feed_forward(_Ctx(), h, gu, down, ids, wts, y, "silu", 0.0, identity=identity > 0)
            x1, x2, o1, o2 = x.clone(), x.clone(), torch.empty(T, K, dtype=bf, device="cuda"), torch.empty(T, K, dtype=bf, device="cuda")
            ops.residual_norm(x1, y, w, 1e-5, then_weight=w2, then_eps=1e-5, out=o1)
            ops.residual_norm(x2, rows, w, 1e-5, then_weight=w2, then_eps=1e-5, out=o2)
            close(x2, x1.cpu(), torch.float32, "residual", 1e-5)
            close(o2, o1.cpu(), bf, "normed", 1e-2)


@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 24, 40), (3, 1, 15, 9), (8, 8, 64, 32), (2, 1, 128, 16), (6, 2, 16, 12), (5, 5, 32, 8)])
@pytest.mark.parametrize("turned,factor,layout", [(8, 1.3, "half"), (14, 1.0, "half"), (0, 1.0, "half"), (6, 0.9, "interleaved"), (16, 1.1, "half")])
def test_biased_normed_maps_into_pages(both, H, G, dim, vdim, turned, factor, layout):
    """A bias, the norm, a rotation of the first channels at positions across pages, two maps to a cached row."""
    from garuda_b200.parts.rotary import RotaryParams
    ops, ref, dt = both
    if turned > dim:
        pytest.skip("not that many channels")
    ps, lead = 8, 4 if dim % 16 == 0 else 1           # (rows that start on 16 bytes and rows that do not)
    b, table, pages = step_batch([5, 1, 60, 2], [0, 62, 3, 5], [2, 0, 3, 1], ps)
    bg = batches(b)[0].batch
    rot = RotaryParams(100.0, turned, layout == "interleaved", tuple(1.0 / (i + 1.5) for i in range(turned // 2)), factor) if turned else None
    T, cols = b.num_tokens, 2 * (H + G) * dim + G * vdim
    row, bias, qw, kw = rnd(T, cols + lead + 4 - (cols + lead) % 4, seed=1), rnd(cols, seed=2), rnd(2 * H, dim, seed=3), rnd(dim, seed=4)
    kp, vp, q = torch.zeros(pages, G, ps, 2 * dim, dtype=dt), torch.zeros(pages, G, ps, vdim, dtype=dt), torch.zeros(T, 2 * H, dim, dtype=dt)
    kg, vg, qg = kp.cuda(), vp.cuda(), q.cuda()
    c = (lead, lead + 2 * H * dim, lead + 2 * (H + G) * dim)
    ref.qk_norm_rope_append(row, c, q, kp, vp, b.positions, b.token_req, table, 2 * H, 2 * G, dim, vdim, qw, kw, 1e-5, rot, ps, bias=bias, maps=2)
    ops.qk_norm_rope_append(row.cuda(), c, qg, kg, vg, bg.positions, bg.token_req, table.cuda(), 2 * H, 2 * G, dim, vdim, qw.cuda(), kw.cuda(), 1e-5,
                            rot, ps, bias=bias.cuda(), maps=2)
    for got, want, what in ((qg, q, "queries"), (kg, kp, "keys"), (vg, vp, "values")):
        close(got, want, dt, f"{what}, {turned} turned", 1e-2 if dt == torch.bfloat16 else 1e-5)


def test_other_kernels_refuse_a_number_on_the_rotation(both):
    from garuda_b200.kernels.ops import KernelError
    from garuda_b200.parts.rotary import RotaryParams
    ops, _, _ = both
    x, pos = torch.zeros(3, 2, 8, device="cuda"), torch.arange(3, dtype=torch.int32, device="cuda")
    with pytest.raises(KernelError, match="cosines"):
        ops.rope_inplace(x, pos, RotaryParams(1e4, 8, False, None, 1.2))


ATT_SIZES = [(6, 2, 10, 13), (4, 2, 32, 64), (2, 1, 64, 128), (3, 3, 48, 96), (8, 1, 16, 16), (16, 1, 16, 112), (40, 1, 32, 16), (2, 2, 128, 80), (1, 1, 200, 300)]


@pytest.mark.parametrize("H,G,dim,vdim", ATT_SIZES)
@pytest.mark.parametrize("window,gated", [(0, True), (7, False), (100, True)])
@pytest.mark.parametrize("lens,starts", [([5, 1, 70, 130], [0, 300, 3, 61]), ([1, 1, 1], [0, 63, 511]), ([2, 2], [126, 400]), ([200], [0])])
def test_differential_attention(both, H, G, dim, vdim, window, gated, lens, starts):
    """Prompt tiles, decoded tokens over many shares of the keys, both in one step; every cache byte that nobody may
    read is NaN, pages in front of a window are given back."""
    ops, ref, dt = both
    ps = 16
    b, table, pages = step_batch(lens, starts, list(range(len(lens))), ps)
    if window:
        for r in range(b.num_requests):
            first = max(0, int(b.kv_lens[r]) - lens[r] + 1 - window) // ps
            table[r, :first] = -1
    ctx_g, ctx_r = batches(b)
    kp, vp = torch.full((pages, G, ps, 2 * dim), float("nan"), dtype=dt), torch.full((pages, G, ps, vdim), float("nan"), dtype=dt)
    for r in range(b.num_requests):
        for j in range(int(b.kv_lens[r])):
            page = int(table[r, j // ps])
            if page >= 0:
                kp[page, :, j % ps] = rnd(G, 2 * dim, seed=1000 * r + j).to(dt)
                vp[page, :, j % ps] = rnd(G, vdim, seed=5000 + 1000 * r + j).to(dt)
    q, gate = rnd(b.num_tokens, H, 2 * dim, dtype=dt, seed=7), rnd(b.num_tokens, H + 3, seed=8)
    want, got = torch.zeros(b.num_tokens, H * vdim, dtype=dt), torch.zeros(b.num_tokens, H * vdim, dtype=dt, device="cuda")
    args = (1.0 / dim ** 0.5, window, ps, 0.8, 0.6, 1e-5)
    ref.differential_attention(ctx_r, q, kp, vp, table, want, *args, gate[:, 2:2 + H] if gated else None)
    ops.differential_attention(ctx_g, q.cuda(), kp.cuda(), vp.cuda(), table.cuda(), got, *args, gate.cuda()[:, 2:2 + H] if gated else None)
    # (a difference of two rows that nearly cancel is divided by its small root mean square: bfloat16 scores
    # and probabilities show more there than in an ordinary attention)
    close(got, want, dt, f"attention {lens}", 6e-2 if dt == torch.bfloat16 else 5e-5)


MEMORY_SIZES = [(3, 7, 11), (2, 64, 32), (1, 16, 48), (2, 128, 64), (1, 256, 128), (4, 32, 16), (2, 300, 20), (1, 80, 600), (5, 20, 16)]


def _memory(H, D, P, T, slots, seed=1):
    """Rows, gates and states: input gates on both sides of zero, forget gates from nearly closed to nearly open."""
    HP, HD = H * P, H * D
    act, gates = rnd(T, HP + 2 * HD, seed=seed), rnd(T, HP + 2 * H, scale=3.0, seed=seed + 1)
    w = dict(b_i=rnd(H, scale=2.0, seed=seed + 2), b_f=torch.linspace(-3.0, 9.0, H), norm=rnd(HP, seed=seed + 3))
    n = HP * D + HD + H
    state = rnd(slots, (n + 3) // 4 * 4, seed=seed + 4)
    state[:, HP * D + HD:n] = state[:, HP * D + HD:n].abs() * 2 - 1.5          # m
    return act, gates, w, state, HP, n


def _run_memory(ops, ctx, act, gates, w, state, H, D, P, out, dev):
    single = ctx.batch.max_q_len == 1
    rows = act.to(dev) if single else act.to(out.dtype).to(dev)
    ops.matrix_memory(ctx, rows, gates.to(dev), w["b_i"].to(dev), w["b_f"].to(dev), 8.0, w["norm"].to(dev), D ** -0.5, 1e-5, state, H, D, P, out)


@pytest.mark.parametrize("H,D,P", MEMORY_SIZES)
@pytest.mark.parametrize("lens,slots", [([5, 1, 200, 64, 65], [2, 0, 5, 3, 1]), ([1, 1, 1], [1, 4, 0]), ([2, 3], [0, 1]), ([129], [3]), ([17, 23, 1], [3, 0, 1]), ([1], [2])])
def test_matrix_memory_steps(both, H, D, P, lens, slots):
    """Mixed steps (single tokens beside portions that end inside a chunk, at its edge and just behind), single
    tokens alone, short portions; states that are not zero; a slot nobody uses is left as it is, NaN and all."""
    ops, ref, dt = both
    b, _, _ = step_batch(lens, [3] * len(lens), slots, 8)
    ctx_g, ctx_r = batches(b)
    T = b.num_tokens
    act, gates, w, state, HP, n = _memory(H, D, P, T, 7)
    state[6] = float("nan")
    want, s_want = torch.zeros(T, HP, dtype=dt), state.clone()
    _run_memory(ref, ctx_r, act, gates, w, s_want, H, D, P, want, "cpu")
    got, s_got = torch.zeros(T, HP, dtype=dt, device="cuda"), state.clone().cuda()
    _run_memory(ops, ctx_g, act, gates, w, s_got, H, D, P, got, "cuda")
    close(got, want, dt, f"matrix memory {lens}", 1e-2 if dt == torch.bfloat16 else 1e-4)
    assert torch.isnan(s_got[6]).all()
    # the state takes the rounded activations in both: what differs is 32-bit rounding
    for a, z, what in ((0, HP * D, "S"), (HP * D, n - H, "n"), (n - H, n, "m")):
        close(s_got[:6, a:z], s_want[:6, a:z], torch.float32, f"its {what}", 5e-5)


def test_matrix_memory_padding_rows_touch_no_state(both):
    ops, ref, dt = both
    H, D, P = 2, 64, 32
    b, _, _ = step_batch([1, 1, 1, 1], [3, 3, 0, 0], [1, 0, -1, -1], 8)
    ctx_g, ctx_r = batches(b)
    act, gates, w, state, HP, n = _memory(H, D, P, 4, 3)
    want, s_want = torch.zeros(4, HP, dtype=dt), state.clone()
    _run_memory(ref, ctx_r, act, gates, w, s_want, H, D, P, want, "cpu")
    got, s_got = torch.zeros(4, HP, dtype=dt, device="cuda"), state.clone().cuda()
    _run_memory(ops, ctx_g, act, gates, w, s_got, H, D, P, got, "cuda")
    close(got[:2], want[:2], dt, "rows with a slot", 1e-2 if dt == torch.bfloat16 else 1e-4)
    assert torch.equal(s_got[2].cpu(), state[2]) and torch.isfinite(got).all()


@pytest.mark.parametrize("H,D,P", [(2, 64, 32), (2, 128, 64), (1, 256, 128)])
def test_chunks_on_the_tensor_cores_keep_32_bit_memories(H, D, P):
    """1,500 tokens through the chunked kernel, through the token-by-token kernel and in steps of many sizes, single tokens
    among them: the same rounded activations enter all, so memories, normalizers and read-outs agree to 32-bit rounding
    (a memory or a weight rounded to bfloat16 anywhere would differ by 2^-9)."""
    from garuda_b200.kernels.ops import CudaOps
    ops = CudaOps("cuda:0")
    T = 1500
    act, gates, w, state, HP, n = _memory(H, D, P, T, 2)
    w["b_f"] = torch.linspace(4.0, 8.0, H)            # long memories among them
    gates[:, HP + H:] *= 0.5
    outs_by, states = [], []
    for cut in ([T], [T], (1, 2, 23, 24, 64, 65, 1, 300, 1, 1019)):
        st, outs, at = state.clone().cuda(), [], 0
        ops.SSD_CHUNK_TOKENS = 10 ** 9 if len(states) == 1 else 24
        for m in cut:
            b, _, _ = step_batch([m], [at], [1], 8)
            ctx, _ = batches(b)
            out = torch.zeros(m, HP, dtype=torch.bfloat16, device="cuda")
            _run_memory(ops, ctx, act[at:at + m], gates[at:at + m], w, st, H, D, P, out, "cuda")
            outs.append(ctx.ws.get("memory_y", (m, HP), torch.float32).clone() if m > 1 else torch.zeros(1, HP, device="cuda"))
            at += m
        assert at == T
        outs_by.append(torch.cat(outs))
        states.append(st)
    single = (outs_by[2] == 0).all(-1)
    for k in (1, 2):
        close(outs_by[k][~single], outs_by[0][~single].cpu(), torch.float32, "read-outs", 2e-5)
        for a, z in ((0, HP * D), (HP * D, n - H), (n - H, n)):
            close(states[k][1, a:z], states[0][1, a:z].cpu(), torch.float32, "states", 3e-5)
    assert torch.equal(states[0][0].cpu(), state[0])


# ---------------------------------------------------------------------------- the engine, replayed
def check(got, ref, dtype, what, name):
    """Per position, the largest difference as a fraction of the largest logit. 32-bit: every position
    within 2e-4 (sums in another order than the 64-bit plain model's). bfloat16: nine positions in ten
    within 0.06 and the median of sixteen and more within 0.015, the rest finite: with sharpened random weights a router's
    close call, a sharp softmax or two maps that nearly cancel turn the rounding of an input into a large change at a
    few positions, in the plain model itself; a fault of a kernel, a mask or a state shows at most positions."""
    scale = float(np.abs(ref).max())
    assert got.shape == ref.shape and np.isfinite(got).all(), what
    err = np.abs(got - ref).max(-1) / scale
    helpers.OBSERVED[f"{name}/{dtype}"] = max(helpers.OBSERVED.get(f"{name}/{dtype}", 0.0), float(np.median(err)))
    if dtype == "float32":
        assert err.max() <= 2e-4, f"{what}: {err.max():.3e} of the largest logit at position {int(err.argmax())}"
        return
    over = int((err > 0.06).sum())
    assert over <= max(1, len(err) // 10), f"{what}: {over} of {len(err)} positions beyond 0.06 (largest {err.max():.3e})"
    assert len(err) < 16 or np.median(err) <= 0.015, f"{what}: median {np.median(err):.3e}"


@pytest.fixture(scope="module", params=[(n, d) for n in CASES for d in ("float32", "bfloat16")], ids=lambda p: f"{p[0]}-{p[1]}")
def run(request):
    name, dtype = request.param
    tr = TraceRunner(model_dir(name, STORE[dtype]), dtype, max_tokens=4 * up64(130), extra=["--page-size", "16"])
    yield name, dtype, tr
    assert tr.close() == 0


def test_whole(run):
    name, dtype, tr = run
    for n, seed in ((1, 1), (2, 2), (17, 3), (130, 4)):
        toks = random_tokens(name, n, seed)
        out = tr.step([("w", toks, range(n))], end=["w"])
        check(out, plain_logits(name, STORE[dtype], toks), dtype, f"whole, {n} tokens", name)


def test_prompt_then_token_by_token(run):
    name, dtype, tr = run
    toks = random_tokens(name, 120, 7)
    ref = plain_logits(name, STORE[dtype], toks)
    outs = [tr.step([("d", toks[:39], [38])])]
    for i in range(39, 120):                      # the windows pass over decoded tokens
        outs.append(tr.step([("d", [toks[i]], [0])], end=["d"] if i == 119 else []))
    check(np.concatenate(outs), ref[38:], dtype, "decode after a prompt", name)


def test_long_decoding_from_the_first_token(run):
    name, dtype, tr = run
    toks = random_tokens(name, 100, 9)
    ref = plain_logits(name, STORE[dtype], toks)
    got = np.concatenate([tr.step([("l", [t], [0])], end=["l"] if i == 99 else []) for i, t in enumerate(toks)])
    check(got[:4], ref[:4], dtype, "first tokens", name)
    check(got, ref, dtype, "long decoding", name)


def test_portions_down_to_two_tokens(run):
    name, dtype, tr = run
    toks = random_tokens(name, 118, 11)
    ref = plain_logits(name, STORE[dtype], toks)
    cuts = [7, 2, 19, 3, 2, 16, 2, 31, 1, 15, 2, 18]
    pos, outs = 0, []
    for i, c in enumerate(cuts):
        outs.append(tr.step([("p", toks[pos:pos + c], range(c))], end=["p"] if i == len(cuts) - 1 else []))
        pos += c
    assert pos == 118
    check(np.concatenate(outs), ref, dtype, "portions", name)


def test_mixed_requests_reusing_pages_and_slots(run):
    name, dtype, tr = run
    lens = [90, 33, 128, 21, 64, 2, 75]
    toks = [random_tokens(name, n, 20 + i) for i, n in enumerate(lens)]
    refs = [plain_logits(name, STORE[dtype], t) for t in toks]
    pool = 4 * up64(130) - 128
    fed, got = [0] * len(lens), [[] for _ in lens]
    live, waiting = [], list(range(len(lens)))
    rng = np.random.default_rng(1)
    most = 0
    while live or waiting:
        while waiting and len(live) < 4 and sum(up64(lens[i]) for i in live) + up64(lens[waiting[0]]) <= pool:
            live.append(waiting.pop(0))
        most = max(most, len(live))
        entries, ended = [], []
        active = [i for i in live if rng.random() > 0.15] or live[:1]        # now and then a request sits a step out
        for i in active:
            left = lens[i] - fed[i]
            n = 1 if left <= 12 else int(min(left - 12, rng.integers(2, 24)))
            entries.append((f"m{i}", toks[i][fed[i]:fed[i] + n], range(n)))
            if fed[i] + n == lens[i]:
                ended.append(f"m{i}")
        out = tr.step(entries, end=ended)
        row = 0
        for (_, t, _), i in zip(entries, active):
            got[i].append(out[row:row + len(t)])
            row += len(t)
            fed[i] += len(t)
            if fed[i] == lens[i]:
                live.remove(i)
    assert most == 4
    for i in range(len(lens)):
        check(np.concatenate(got[i]), refs[i], dtype, f"mixed, request {i}", name)


def test_every_way_of_cutting_gives_the_same_logits_in_32_bit(run):
    name, dtype, tr = run
    if dtype != "float32":
        pytest.skip("compared against the plain model in bfloat16")
    toks = random_tokens(name, 80, 31)
    whole = tr.step([("x", toks, range(80))], end=["x"])
    parts = [tr.step([("y", toks[:50], range(50))])]
    parts += [tr.step([("y", [t], [0])]) for t in toks[50:79]]
    parts.append(tr.step([("y", [toks[79]], [0])], end=["y"]))
    assert np.abs(np.concatenate(parts) - whole).max() <= 3e-5 * max(1.0, np.abs(whole).max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [40, 64, 500])
def test_a_key_just_inside_and_just_outside_the_window(dtype, window, tmp_path):
    """Token 0 once, the last seen and the first not seen position in front of queries for it (token 1) in a portion and
    decoded, at places on page borders and beside them; the plain model's logits with and without it are others altogether,
    or the same."""
    d, cfg = edge_model(str(tmp_path / "m"), STORE[dtype], window=window)
    W = helpers.folder_weights(d)
    tr = TraceRunner(d, dtype, max_tokens=up64(660), extra=["--page-size", "16"])
    base = np.random.default_rng(5).integers(2, 80, 640)
    limit = 1e-4 if dtype == "float32" else 0.04
    for k, query in enumerate((window + 7, window + 15, window + 16, window + 31, window + 64)):
        for back, seen in ((window - 1, True), (window, False)):
            toks = base[:query + 4].copy()
            toks[query], toks[query - back] = 1, 0
            ref = rp.forward(cfg, W, toks).astype(np.float32)
            without = toks.copy()
            without[query - back] = base[query - back]
            other = rp.forward(cfg, W, without)
            scale = np.abs(ref).max()
            change = np.abs(other[query] - ref[query]).max() / scale
            assert change > 0.2 if seen else change < 1e-6
            toks = toks.tolist()
            out = tr.step([(f"p{k}{back}", toks, [query - 1, query, query + 1])], end=[f"p{k}{back}"])
            assert np.abs(out - ref[query - 1:query + 2]).max() <= limit * scale, f"portion, {back} back at {query}"
            tr.step([(f"d{k}{back}", toks[:query - 2], [])])
            out = np.concatenate([tr.step([(f"d{k}{back}", [t], [0])], end=[f"d{k}{back}"] if i == 3 else []) for i, t in enumerate(toks[query - 2:query + 2])])
            assert np.abs(out - ref[query - 2:query + 2]).max() <= limit * scale, f"decoded, {back} back at {query}"
    assert tr.close() == 0


def test_a_long_request_whose_early_tokens_reach_the_end():
    """700 tokens; the last logits follow the plain model in both dtypes, and they change with token 3 (through the memories:
    the windows have long passed)."""
    name = "RB"
    toks = random_tokens(name, 700, 3)
    for dtype in ("float32", "bfloat16"):
        ref = plain_logits(name, STORE[dtype], toks)
        tr = TraceRunner(model_dir(name, STORE[dtype]), dtype, max_tokens=up64(700))
        tr.step([("a", toks[:300], [])])
        out = tr.step([("a", toks[300:], range(390, 400))], end=["a"])
        check(out, ref[690:], dtype, "the end of 700 tokens", name)
        if dtype == "float32":
            other = list(toks)
            other[3] = (toks[3] + 1) % CASES[name][0]["vocab"]
            alt = tr.step([("b", other, range(690, 700))], end=["b"])
            assert np.abs(alt - out).max() > 1e-4 * np.abs(out).max()
        assert tr.close() == 0


@pytest.mark.parametrize("name,dtype", [("RB", "float32"), ("RB", "bfloat16"), ("RA", "bfloat16")])
def test_greedy_generation_through_the_engine(name, dtype):
    from garuda_b200 import Engine, SamplingParams
    cfg, w = CASES[name][0], weights(name, STORE[dtype])
    e = Engine(model_dir(name, STORE[dtype]), dtype=dtype, context=256, kv_tokens=1024, max_concurrent=4)
    assert e.model.graph_safe
    prompts = [random_tokens(name, n, 70 + n) for n in (5, 40, 1, 23, 64)]
    res = e.generate(prompts, SamplingParams.greedy(max_tokens=12))
    assert e.runner.graphs.replays > 0
    for p, r in zip(prompts, res):
        assert r.finish_reason == "length" and len(r.tokens) == 12
        seq = list(p)
        for tok in r.tokens:
            logits = rp.forward(cfg, w, seq)[-1]
            slack = (1e-4 if dtype == "float32" else 0.08) * float(np.abs(logits).max())
            assert logits[tok] >= float(logits.max()) - slack, f"token {tok} has logit {logits[tok]}, the best is {logits.max()}"
            seq.append(tok)


# ---------------------------------------------------------------------------- configurations drawn at random
def _random_config(rng):
    def pick(xs):
        return xs[int(rng.integers(0, len(xs)))]

    def attention():
        g, dim = pick([1, 2, 3]), pick([8, 12, 15, 32, 48, 64])
        m = {"heads": g * pick([1, 2, 4]), "kv_heads": g, "dim": dim, "vdim": pick([8, 20, 32, 64, 128]), "scale": pick([0.2, 0.4, 0.7]), "diff": pick([0.2, 0.5, 0.8])}
        if pick([True, True, False]):
            m["mask"] = {"size": pick([1, 5, 16, 33, 64, 1000])}
        if pick([True, True, False]):
            m["rot"] = {"base": pick([100.0, 10000.0]), "dims": pick([2, 4, dim // 2 // 2 * 2, dim // 2 * 2])}
            if pick([True, False]):
                m["rot"]["scaling"] = {"factor": pick([1.0, 2.0, 16.0]), "original": pick([32, 1000]), "fast": pick([4.0, 32.0]), "slow": pick([0.5, 1.0])}
        return {"type": "attention", "mixer": m}

    def memory():
        return {"type": "mlstm", "mixer": {"heads": pick([1, 2, 3, 5]), "dim": pick([4, 16, 33, 64, 128, 144]), "vdim": pick([4, 16, 24, 32, 64, 96]), "gate_cap": pick([1.0, 8.0, 15.0])}}

    def mlp():
        if pick([True, True, True, False]) is False:
            return None
        size, count = pick([1, 2, 3, 4]), pick([1, 2, 4])
        keep, choices = int(rng.integers(1, count + 1)), size * count
        identity = int(rng.integers(0, choices))
        f = {"kind": "moe", "expert": {"ff": pick([8, 24, 64])}, "router": {"experts": choices - identity, "top": int(rng.integers(1, size * keep + 1))}}
        if identity:
            f["router"]["identity"] = identity
        if count > 1 or pick([True, False]):
            f["router"]["groups"] = {"count": count, "keep": keep}
        if pick([True, False]):
            f["shared"] = {"ff": pick([8, 40, 64])}
        return f

    layers = [dict(attention() if pick([True, False]) else memory(), mlp=mlp()) for _ in range(pick([1, 2, 3, 4]))]
    cfg = {"architecture": "Ruvalix", "vocab": pick([50, 97, 300, 1000]), "width": pick([40, 64, 72, 136, 256]), "norm": {"eps": pick([1e-5, 1e-6])}, "layers": layers}
    if pick([True, True, False]):
        start = int(rng.integers(0, len(layers)))
        cfg["loop"] = {"start": start, "stop": int(rng.integers(start + 1, len(layers) + 1)), "times": pick([1, 2, 3])}
    return cfg


@pytest.mark.parametrize("seed", [2, 7])
def test_configurations_drawn_at_random(seed, tmp_path):
    rng = np.random.default_rng(seed)
    for k in range(3):
        cfg = _random_config(rng)
        for dtype in ("float32", "bfloat16"):
            d = write(str(tmp_path / f"m{k}{dtype}"), cfg, seed * 10 + k, STORE[dtype])
            w = helpers.folder_weights(d)
            a, b = rng.integers(0, cfg["vocab"], 70).tolist(), rng.integers(0, cfg["vocab"], 45).tolist()
            ra, rb = rp.forward(cfg, w, a).astype(np.float32), rp.forward(cfg, w, b).astype(np.float32)
            tr = TraceRunner(d, dtype, max_tokens=2 * up64(70), extra=["--page-size", "16"])
            check(tr.step([("w", a, range(70))], end=["w"]), ra, dtype, f"seed {seed}.{k}: whole", "random")
            outs_a, outs_b = [tr.step([("a", a[:40], range(40)), ("b", b[:3], range(3))])], []
            outs_b.append(outs_a[0][40:])
            outs_a[0] = outs_a[0][:40]
            o = tr.step([("b", b[3:30], range(27)), ("a", a[40:42], range(2))])
            outs_b.append(o[:27])
            outs_a.append(o[27:])
            for i in range(15):
                o = tr.step([("a", [a[42 + i]], [0]), ("b", [b[30 + i]], [0])], end=["b"] if i == 14 else [])
                outs_a.append(o[:1])
                outs_b.append(o[1:])
            outs_a.append(tr.step([("a", a[57:], range(13))], end=["a"]))
            check(np.concatenate(outs_a), ra, dtype, f"seed {seed}.{k}: request a", "random")
            check(np.concatenate(outs_b), rb, dtype, f"seed {seed}.{k}: request b", "random")
            assert tr.close() == 0


def test_command_line_generates_with_sampling(tmp_path):
    """`garuda generate` on a folder of this design: greedy tokens are the plain model's, and a
    sampled run with a seed (temperature, top-k, top-p through the engine's sampler) repeats itself."""
    name = "RA"
    d = model_dir(name)
    cfg = tmp_path / "config.toml"
    prompt = random_tokens(name, 11, 5)
    exe = [sys.executable, os.path.join(helpers.ROOT, "bin", "garuda")]

    def generate(sampling, *more):
        cfg.write_text(f'[model]\npath = "{d}"\ndtype = "float32"\ncontext = 128\n[memory]\npage_size = 16\n[sampling]\n{sampling}')
        out = subprocess.run(exe + ["--config", str(cfg), "generate", "--prompt-ids", ",".join(map(str, prompt)), *more],
                             capture_output=True, text=True)
        assert out.returncode == 0, out.stderr
        return json.loads(out.stdout.strip().splitlines()[-1])

    rec = generate("temperature = 0.0\nmax_tokens = 6\n")
    seq = list(prompt)
    for _ in range(6):
        seq.append(int(np.argmax(rp.forward(CASES[name][0], weights(name), seq)[-1])))
    assert rec["tokens"] == seq[len(prompt):] and rec["finish_reason"] == "length"
    a = generate("temperature = 0.9\ntop_k = 20\ntop_p = 0.9\nmax_tokens = 8\n", "--seed", "4")
    b = generate("temperature = 0.9\ntop_k = 20\ntop_p = 0.9\nmax_tokens = 8\n", "--seed", "4")
    assert a["tokens"] == b["tokens"] and len(a["tokens"]) == 8

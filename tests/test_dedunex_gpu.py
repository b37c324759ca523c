"""Dedunex on the GPU: every new kernel and every kernel option alone against plain torch in float64, every mechanism
alone as a one-layer model, and whole models through the step function, cut into steps every way, against the plain
implementation (tests/plain_dedunex.py).  Test weights are made so that faults show (dedunex_util.write_model); where
random values would still hide one (a key at the edge of a window, a token far back), the test builds queries and keys,
or the prompts, by hand."""
import json
import math
import random

import pytest
import torch

from dedunex_util import TOL, assert_close, config, dense, diff_layer, gru_layer, latent_layer, rel_err, row_errs, write_model
from test_mulavik_gpu import _paged, step_ctx, toks

pytestmark = pytest.mark.gpu

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DEV = "cuda"


# =============================================================================== kernels alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,groups", [(40, 1), (40, 5), (264, 2), (36, 4), (1536, 1), (2048, 2), (6000, 1), (30, 10), (4096, 2)])
def test_norm_in_groups_with_a_vector_added_and_with_rows_picked(C, groups, dtype):
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(C + groups)
    dt, T, R, eps = DT[dtype], 9, 12, 3e-5
    x0, w, add = torch.randn(R, C, device=DEV) * 3, torch.rand(C, device=DEV) + 0.5, torch.randn(C, device=DEV)
    tol = 2e-6 if dtype == "float32" else 1e-2

    def norm(v):
        p = v.double().view(-1, groups, C // groups)
        return (p / torch.sqrt((p ** 2).mean(-1, keepdim=True) + eps)).view(-1, C) * w.double()
    close = lambda a, b: float(((a.double() - b) / (b.abs() + 1)).abs().max()) < tol
    x, out = x0.clone(), torch.full((R, C), 7.0, device=DEV, dtype=dt)
    ops.group_norm(x, w, groups, eps, out, T)
    assert close(out[:T], norm(x0[:T])) and torch.equal(x, x0) and float(out[T:].float().min()) == 7.0
    ops.group_norm(x, w, groups, eps, out, T, add=add)
    want = x0[:T] + add
    assert close(out[:T], norm(want)) and torch.equal(x[:T], want) and torch.equal(x[T:], x0[T:])
    ops.group_norm(x, None, groups, eps, None, T, add=add)          # the sum alone
    assert torch.equal(x[:T], want + add) and torch.equal(x[T:], x0[T:])
    rows = torch.tensor([11, 0, 5], dtype=torch.int32, device=DEV)
    ops.group_norm(x0, w, groups, eps, out, 3, rows=rows)
    assert close(out[:3], norm(x0[rows.long()]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,groups", [(40, 2), (30, 3), (768, 1), (1024, 4)])
def test_embedding_with_a_norm_behind_it(C, groups, dtype):
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(C)
    table = torch.randn(50, C, device=DEV).to(DT[dtype])
    w, eps = torch.rand(C, device=DEV) + 0.5, 2e-4
    tokens = torch.tensor([3, 49, -3, 0, 3], dtype=torch.int32, device=DEV)          # -3: what was sampled for slot 2
    feedback = torch.tensor([9, 8, 17, 6], dtype=torch.int32, device=DEV)
    out = torch.full((7, C), 7.0, device=DEV)
    ops.embed_group_norm(tokens, table, out, w, groups, eps, feedback=feedback, scale=1.5)
    p = (table[[3, 49, 17, 0, 3]].double() * 1.5).view(5, groups, C // groups)
    want = (p / torch.sqrt((p ** 2).mean(-1, keepdim=True) + eps)).view(5, C) * w.double()
    assert float((out[:5].double() - want).abs().max()) < 5e-6 and float(out[5:].min()) == 7.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [1, 31, 64, 100, 257])
def test_recurrent_unit_carries_its_state_in_the_slot(width, dtype):
    """Portions of 1 to 1500 rows over shuffled slots, rows of no request behind them; channels that forget at once and
    channels that remember for thousands of rows."""
    from nanoinfer_b200.kernels import ops

    g = torch.Generator().manual_seed(width)
    n_slots, pad = 5, 3
    state = torch.zeros(n_slots, width + pad, device=DEV)
    state[:, width:] = 3.0
    ref = torch.zeros(n_slots, width, dtype=torch.float64)
    slow = torch.rand(width, generator=g) * 12.0 - 9.0
    tol = 2e-5 if dtype == "float32" else 1e-2
    for step, (rows, slots) in enumerate([([5, 1, 19], [3, 0, 4]), ([1, 1, 1], [4, 3, 0]), ([2, 1500], [0, 1]), ([130, 127, 3], [4, 3, 1]),
                                          ([1], [2]), ([1024, 1025], [0, 2])]):
        T = sum(rows)
        ctx = step_ctx(rows, [p for n in rows for p in range(n)], slots=slots, n_pad=2)
        proj = torch.randn(T + 2, 3 * width + 9, generator=g) * 2
        offs = (2 * width + 5, 1, width + 3)
        proj[:, offs[0]:offs[0] + width] += slow
        proj[0, offs[1]] = 0.0                                        # (u = 0 takes the branch of u >= 0)
        out = torch.full((T + 2, width + 4), 7.0, device=DEV, dtype=DT[dtype])
        ops.min_gru(proj.to(DEV), offs, width, state, ctx, out)
        at = 0
        for n, s in zip(rows, slots):
            z, u, gg = (proj[at:at + n, o:o + width].double() for o in offs)
            z, cand = torch.sigmoid(z), torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
            want = torch.zeros(n, width, dtype=torch.float64)
            for t in range(n):
                ref[s] = (1 - z[t]) * ref[s] + z[t] * cand[t]
                want[t] = ref[s] * gg[t] * torch.sigmoid(gg[t])
            got = out[at:at + n, :width].double().cpu()
            assert float(((got - want) / (want.abs() + 1)).abs().max()) < tol, (step, s)
            at += n
        assert float(out[T:].float().min()) == 7.0 and float(out[:, width:].float().min()) == 7.0
        assert float((state[:, :width].double().cpu() - ref).abs().max()) < 2e-5 and float(state[:, width:].min()) == 3.0


def _turn_halves(x, pos, dims, freqs, amp):
    """x [n, heads, dim] float64."""
    if not dims:
        return x
    half = dims // 2
    ang = pos.double()[:, None] * freqs
    c, s = (torch.cos(ang) * amp)[:, None], (torch.sin(ang) * amp)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dim,vdim,hd,rot,norm", [(4, 2, 16, 40, 48, 8, True), (3, 1, 24, 20, 48, 24, True), (2, 2, 7, 33, 48, 0, False),
                                                      (1, 1, 64, 128, 128, 32, True), (6, 3, 128, 256, 256, 128, True), (2, 1, 100, 10, 208, 2, False)])
def test_two_maps_normed_turned_and_laid_into_the_cached_row(H, G, dim, vdim, hd, rot, norm, dtype):
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.base import POSITIONS

    torch.manual_seed(H + dim)
    dt, page, eps = DT[dtype], 16, 3e-5
    rows, positions = [5, 1, 3], [0, 1, 2, 3, 4, 40, 14, 15, 16]
    ctx = step_ctx(rows, positions, n_pad=2)
    T = ctx.n_rows
    nq, nk, nv = H * 2 * dim, G * 2 * dim, G * vdim
    src = torch.randn(T, nq + nk + nv + 7, device=DEV) * 2
    offs = (3, 3 + nq, 5 + nq + nk)
    wq, wk = (torch.rand(dim, device=DEV) + 0.5, torch.rand(dim, device=DEV) + 0.5) if norm else (None, None)
    pos_part = POSITIONS.build("rotary_halves", base=700.0, dims=rot, scaling=dict(factor=3.0, original=60, fast=4.0, slow=0.5)) if rot else None
    if rot:
        pos_part.prepare(dt, torch.device(DEV))
    amp = pos_part.amplitude if rot else 1.0
    table = torch.tensor([[3, -1, -1], [5, 0, 4], [2, 1, -1]], dtype=torch.int32, device=DEV)
    cache = torch.full((6, 2, G, page, hd), 9.0, device=DEV, dtype=dt)
    q_out = torch.full((T, H * 2 * hd + 8), 7.0, device=DEV, dtype=dt)
    ops.norm_rope_maps_append(src, offs, H, G, 2, dim, vdim, wq, wk, eps, rot, pos_part.freqs if rot else None, amp, ctx,
                              q_out[:, :H * 2 * hd], cache, table)
    assert int(ctx.status.item()) == 0
    s = src.double().cpu()
    rms = lambda v, w: v / torch.sqrt((v ** 2).mean(-1, keepdim=True) + eps) * w.double().cpu() if w is not None else v
    pos = torch.tensor(positions + [0, 0])
    fr = torch.tensor(pos_part.frequencies(), dtype=torch.float64) if rot else None
    q = _turn_halves(rms(s[:, offs[0]:offs[0] + nq].view(T, H * 2, dim), wq), pos, rot, fr, amp).view(T, H, 2, dim)
    k = _turn_halves(rms(s[:, offs[1]:offs[1] + nk].view(T, G * 2, dim), wk), pos, rot, fr, amp).view(T, G, 2 * dim)
    v = s[:, offs[2]:offs[2] + nv].view(T, G, vdim)
    tol = 3e-6 if dtype == "float32" else 1e-2
    close = lambda a, b: float(((a.double().cpu() - b) / (b.abs() + 1)).abs().max()) < tol
    want_q = torch.zeros(T, H, 2, hd, dtype=torch.float64)
    want_q[:, :, 0, :dim], want_q[:, :, 1, dim:2 * dim] = q[:, :, 0], q[:, :, 1]
    got_q = q_out[:, :H * 2 * hd].view(T, H, 2, hd)
    assert close(got_q, want_q) and not got_q[:, :, 0, dim:].any() and not got_q[:, :, 1, :dim].any()
    assert float(q_out[:, H * 2 * hd:].float().min()) == 7.0
    entry = [e for e, n in enumerate(rows) for _ in range(n)]
    written = set()
    for t, (e, p) in enumerate(zip(entry, positions)):
        pg, slot = int(table[e, p // page]), p % page
        written.add((pg, slot))
        assert close(cache[pg, 0, :, slot, :2 * dim], k[t]) and close(cache[pg, 1, :, slot, :vdim], v[t])
        assert not cache[pg, 0, :, slot, 2 * dim:].any() and not cache[pg, 1, :, slot, vdim:].any()
    for pg in range(6):
        for slot in range(page):
            if (pg, slot) not in written:
                assert float(cache[pg, :, :, slot].float().min()) == 9.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,hd,vdim", [(3, 48, 40), (1, 16, 3), (4, 128, 128), (2, 256, 255)])
def test_second_map_subtracted_and_the_difference_normed(H, hd, vdim, dtype):
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(hd + vdim)
    T, lam, eps, mul = 11, 0.83, 2e-4, 0.6
    a = torch.randn(T + 1, 2 * H * hd, device=DEV)
    a.view(T + 1, H, 2, hd)[:, :, 1] = a.view(T + 1, H, 2, hd)[:, :, 0] / lam * 1.001 + 0.01 * a.view(T + 1, H, 2, hd)[:, :, 1]  # nearly equal maps
    out = torch.full((T + 1, H * vdim + 3), 7.0, device=DEV, dtype=DT[dtype])
    ops.diff_combine(a, H, vdim, lam, eps, mul, out, T)
    m = a[:T].double().view(T, H, 2, hd)[..., :vdim]
    o = m[:, :, 0] - lam * m[:, :, 1]
    want = (o / torch.sqrt((o ** 2).mean(-1, keepdim=True) + eps) * mul).reshape(T, H * vdim)
    tol = 2e-4 if dtype == "float32" else 1e-2
    assert float(((out[:T, :H * vdim].double() - want) / (want.abs() + 1)).abs().max()) < tol
    assert float(out[T:].float().min()) == 7.0 and float(out[:, H * vdim:].float().min()) == 7.0


def _windowed(q, k, v, scale, pos0, window, cap):
    """q [n, H, d], k, v [m, G, d]: row i stands at position pos0 + i.  float64."""
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros(q.shape[0], H, v.shape[2], dtype=torch.float64)
    j = torch.arange(k.shape[0])
    for h in range(H):
        s = (q[:, h].double() @ k[:, h // (H // G)].double().T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        i = pos0 + torch.arange(q.shape[0])[:, None]
        see = (j <= i) & (i - j < window if window else torch.ones(1, dtype=torch.bool))
        out[:, h] = torch.softmax(s.masked_fill(~see, -math.inf), -1) @ v[:, h // (H // G)].double()
    return out


@pytest.mark.parametrize("hd", [32, 64, 96, 128, 160])
@pytest.mark.parametrize("window,cap", [(0, 0.0), (40, 6.0), (1, 0.0), (130, 50.0)])
def test_attention_leaves_32_bit_results_of_16_bit_heads(hd, window, cap):
    """The bfloat16 kernels with a float32 output (tcgen05, warp-MMA and general for portions, streaming for single
    tokens): nearer to the float64 result than a bfloat16 output could be."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.attention import AttentionPlan

    n_head, n_kv_head, page, dt, scale = 4, 2, 16, torch.bfloat16, 1.2 / math.sqrt(hd)
    lengths, q_rows = [200, 77, 450, 130, 16, 3, 333], [130, 1, 1, 40, 16, 1, 290]
    cache, table, ks, vs, qs = _paged(dt, n_head, n_kv_head, hd, page, lengths, q_rows, seed=hd)
    ctx = step_ctx(q_rows, [p for n, r in zip(lengths, q_rows) for p in range(n - r, n)])
    want = torch.cat([_windowed(qq, k, v, scale, n - r, window, cap) for qq, k, v, n, r in zip(qs, ks, vs, lengths, q_rows)])
    q = torch.cat(qs).view(-1, n_head * hd).to(dt).to(DEV)
    out = torch.full((q.shape[0], n_head * hd), 7.0, device=DEV)
    plan = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0, device=torch.device(DEV))
    ops.attention(q, cache.to(dt).to(DEV), out, table.to(DEV), ctx, n_head, scale, window, plan,
                  extras=ops.AttnExtras(softcap=cap, out32=True))
    assert int(ctx.status.item()) == 0
    err = (out.double().cpu().view(want.shape) - want).abs()
    assert float(err.max()) < 1e-2 and float(err.mean()) < 6e-4        # (P is rounded to 16 bits in the prompt kernels)
    single = [sum(q_rows[:e]) for e, r in enumerate(q_rows) if r == 1]
    assert float(err[single].max()) < 1e-5                              # single tokens: all 32-bit behind the loads


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [1, 2, 40, 150])
@pytest.mark.parametrize("window", [1, 16, 23, 64, 100])
def test_one_matching_key_of_either_map_just_inside_and_just_outside_the_window(window, rows, dtype):
    """Two maps in one cached row: all keys but one of one map are at right angles to that map's query; the one that
    matches carries a value of its own, which shows in that map's output exactly when it lies in the row's window, and
    never in the other map's."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.attention import AttentionPlan

    dt, dim, hd, page, n = DT[dtype], 24, 48, 16, 2 * window + 37 + rows
    for m in (0, 1):
        for far in sorted({n - 1, n - window, n - window - 1, n - window + 1, 0, n - rows, n - rows - window, n - rows - window + 1}):
            if far < 0 or far > n - 1:
                continue
            k = torch.zeros(n, hd)
            k[:, [1, dim + 1]] = 1.0
            k[far, m * dim] = 30.0
            v = torch.zeros(n, hd)
            v[:, 1] = 1.0
            v[far, 1], v[far, 2] = 0.0, 1.0
            q = torch.zeros(rows, 2, hd)
            q[:, 0, 0], q[:, 1, dim] = 1.0, 1.0
            nb = -(-n // page)
            perm = torch.randperm(nb, generator=torch.Generator().manual_seed(far)).tolist()
            cache = torch.zeros(nb, 2, 1, page, hd)
            for b in range(nb):
                c = min(page, n - b * page)
                cache[perm[b], 0, 0, :c], cache[perm[b], 1, 0, :c] = k[b * page:b * page + c], v[b * page:b * page + c]
            ctx = step_ctx([rows], list(range(n - rows, n)))
            plan = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0, device=torch.device(DEV))
            table = torch.tensor([perm], dtype=torch.int32, device=DEV)
            qd, cd = q.view(rows, -1).to(dt).to(DEV), cache.to(dt).to(DEV)
            for layout in (None, (2, dim, hd)):         # (with the layout known, bfloat16 portions take the kernel for wide rows)
                out = torch.zeros(rows, 2 * hd, device=DEV)
                ops.attention(qd, cd, out, table, ctx, 2, 1.0, window, plan, extras=ops.AttnExtras(softcap=25.0, out32=True, layout=layout))
                for i in (0, rows - 1):
                    p = n - rows + i
                    visible = 0 <= p - far < window
                    found, other = float(out[i, m * hd + 2]) > 0.9, float(out[i, (1 - m) * hd + 2])
                    assert found == visible, f"map {m}, key {far}, row at {p}: visible {visible}, found {found}"
                    assert other < (1.01 if window == 1 else 0.55 if window == 2 else 0.2)
            if dtype == "bfloat16" and rows == 1:       # ... and single tokens the grouped kernel, in one piece and in four
                for splits in (1, 4):
                    got = torch.zeros(1, 2 * hd, device=DEV, dtype=dt)
                    assert ops.attention_group_mma(qd, cd, got, hd, table, ctx, plan, 2, 1.0, window, 2 * dim, hd, softcap=25.0, n_splits=splits)
                    assert (float(got[0, m * hd + 2]) > 0.9) == (0 <= n - 1 - far < window)


DIFF_CASES = [(4, 2, 16, 40, 48), (3, 1, 64, 128, 128), (2, 2, 9, 21, 32), (12, 1, 24, 48, 48), (2, 1, 100, 200, 208), (3, 3, 32, 64, 64),
              (1, 1, 128, 256, 256), (5, 5, 40, 8, 80)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,cap", [(0, 0.0), (70, 6.0), (1, 30.0)])
@pytest.mark.parametrize("H,G,dim,vdim,hd", DIFF_CASES)
def test_both_maps_and_their_normed_difference(H, G, dim, vdim, hd, window, cap, dtype):
    """Portions beside single tokens, and single tokens alone with their keys in 1 to 16 pieces: in bfloat16 the tcgen05 kernel
    for wide rows and the grouped one; pages behind the window are gone."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.attention import AttentionPlan

    dt, page, scale, lam, eps, mul = DT[dtype], 16, 1.3 / math.sqrt(dim), 0.7, 1e-4, 0.6
    for lengths, q_rows in (([200, 77, 450, 130, 16, 3, 333], [130, 1, 1, 40, 16, 2, 290]), ([450, 77, 2, 64], [1] * 4), ([1000], [1])):
        cache, table, ks, vs, _ = _paged(dt, 2 * H, G, hd, page, lengths, q_rows, seed=hd)
        cache[:, 0, :, :, 2 * dim:], cache[:, 1, :, :, vdim:] = 0.0, 0.0
        for e, (n, r) in enumerate(zip(lengths, q_rows)):
            for b in range(n // page):
                if window and (b + 1) * page <= n - r - window + 1:
                    table[e, b] = -1
        g = torch.Generator().manual_seed(dim)
        T = sum(q_rows)
        q = torch.randn(T, H, 2, dim, generator=g).to(dt).float()
        laid = torch.zeros(T, H, 2, hd)
        laid[:, :, 0, :dim], laid[:, :, 1, dim:2 * dim] = q[:, :, 0], q[:, :, 1]
        ctx = step_ctx(q_rows, [p for n, r in zip(lengths, q_rows) for p in range(n - r, n)])
        at, want = 0, []
        for n, r, k, v in zip(lengths, q_rows, ks, vs):
            a = [_windowed(q[at:at + r, :, m], k[..., m * dim:(m + 1) * dim], v[..., :vdim], scale, n - r, window, cap) for m in (0, 1)]
            o = a[0] - lam * a[1]
            want.append((o / torch.sqrt((o ** 2).mean(-1, keepdim=True) + eps) * mul).reshape(r, H * vdim))
            at += r
        want = torch.cat(want)
        plan = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0, device=torch.device(DEV))
        qd, cd, td = laid.view(T, -1).to(dt).to(DEV), cache.to(dt).to(DEV), table.to(DEV)
        maps = torch.full((T, 2 * H * hd), 7.0, device=DEV)
        tol = 1e-4 if dtype == "float32" else 5e-2

        def check(out, what):
            assert int(ctx.status.item()) == 0
            err = (out[:, :H * vdim].double().cpu() - want).abs()
            assert float(err.max()) < tol, (lengths, what, float(err.max()))
            assert float(out[:, H * vdim:].float().min()) == 7.0
        out = torch.full((T, H * vdim + 6), 7.0, device=DEV, dtype=dt)
        ops.differential_attention(qd, cd, maps, out, td, ctx, H, dim, vdim, scale, window, cap, lam, eps, mul, plan)
        check(out, "as the step runs it")
        if dtype == "bfloat16" and plan.n_prefill_rows == 0:
            for splits in (1, 2, 4, 8, 16):
                out.fill_(7.0)
                assert ops.attention_group_mma(qd, cd, out, vdim, td, ctx, plan, 2 * H, scale, window, 2 * dim, vdim, softcap=cap,
                                               diff=(lam, eps, mul), n_splits=splits)
                check(out, f"{splits} pieces")


def _latent_reference(q, lat, kv_rank, scale, positions, gate, window=0):
    out = []
    for i, p in enumerate(positions):
        lo = max(0, p - window + 1) if window else 0
        keys = lat[lo:p + 1].double()
        pr = torch.softmax(torch.einsum("hd,jd->hj", q[i].double(), keys) * scale, -1)
        o = pr @ keys[:, :kv_rank]
        out.append(o * torch.sigmoid(gate[i].double())[:, None] if gate is not None else o)
    return torch.stack(out)


def _latent_cache(lats, page, D, seed, dt, gone_behind=None):
    """Pages in a scrambled order; what no request holds is large; ``gone_behind[e]``: entry e's pages wholly behind that
    position were given back."""
    nbs = [-(-len(lat) // page) for lat in lats]
    ids = torch.randperm(sum(nbs) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    table = torch.full((len(lats), max(nbs) + 1), -1, dtype=torch.int32)
    cache = torch.full((sum(nbs) + 3, 1, 1, page, D), 5.0)
    for e, lat in enumerate(lats):
        for b in range(nbs[e]):
            pg = ids.pop()
            c = min(page, len(lat) - b * page)
            cache[pg, 0, 0, :c] = lat[b * page:b * page + c]
            if gone_behind is None or (b + 1) * page > gone_behind[e]:
                table[e, b] = pg
    return cache.to(dt).to(DEV), table.to(DEV)


LATENT_CASES = [(3, 32, 8, 16), (9, 64, 16, 16), (1, 20, 6, 32), (12, 128, 32, 48), (4, 256, 32, 16), (2, 512, 64, 16), (17, 96, 24, 16),
                (5, 256, 64, 32), (40, 16, 8, 16), (2, 8, 0, 16), (3, 200, 40, 16), (2, 256, 128, 16), (3, 336, 48, 16)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("gated,window", [(False, 0), (True, 0), (True, 70), (False, 1)])
@pytest.mark.parametrize("H,kv_rank,rot,page", LATENT_CASES)
def test_latent_attention_every_kernel_with_gates_and_windows(H, kv_rank, rot, page, gated, window, dtype):
    """Portions that start anywhere beside single tokens, and single tokens alone: in bfloat16 the tcgen05 kernel (portions)
    and the warp-MMA one (single tokens, their keys in one to sixteen pieces) where the sizes allow, the general one
    elsewhere; pages behind the window are gone."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.attention import AttentionPlan

    dt, D, scale = DT[dtype], kv_rank + rot, 1.5 / math.sqrt(kv_rank)
    for lengths, q_rows in (([200, 77, 301, 40, 16], [130, 1, 260, 3, 16]), ([300, 1, 77, 64], [1, 1, 1, 1]), ([700], [1]), ([129, 2, 128], [129, 2, 127])):
        g = torch.Generator().manual_seed(H + kv_rank + len(lengths))
        lats = [torch.randn(n, D, generator=g).to(dt).float() for n in lengths]
        first = [max(0, n - r - window + 1) if window else 0 for n, r in zip(lengths, q_rows)]
        cache, table = _latent_cache(lats, page, D, H + kv_rank, dt, first)
        positions = [p for n, r in zip(lengths, q_rows) for p in range(n - r, n)]
        n_pad = 3 if len(lengths) == 5 else 0
        ctx = step_ctx(q_rows, positions, n_pad=n_pad)
        T = len(positions)
        q = torch.randn(T + n_pad, H, D, generator=g).to(dt)
        gate_rows = torch.randn(T + n_pad, H + 5, generator=g) * 2
        out = torch.full((T + n_pad, H * kv_rank + 8), 7.0, device=DEV, dtype=dt)
        plan = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0, device=torch.device(DEV))
        ops.latent_attention(q.to(DEV), cache, out[:, :H * kv_rank], table, ctx, H, kv_rank, scale, window,
                             gate=gate_rows.to(DEV)[:, 2:2 + H] if gated else None, plan=plan)
        assert int(ctx.status.item()) == 0
        at, want = 0, []
        for e, (n, r) in enumerate(zip(lengths, q_rows)):
            want.append(_latent_reference(q[at:at + r], lats[e], kv_rank, scale, range(n - r, n),
                                          gate_rows[at:at + r, 2:2 + H] if gated else None, window))
            at += r
        err = (out[:T, :H * kv_rank].double().cpu() - torch.cat(want).reshape(T, -1)).abs()
        assert float(err.max()) < (2e-5 if dtype == "float32" else 4e-2), (lengths, float(err.max()), int(err.max(1).values.argmax()))
        assert float(out[:, H * kv_rank:].float().min()) == 7.0 and float(out[T:].float().min() if n_pad else 7.0) == 7.0


@pytest.mark.parametrize("window", [0, 33, 64])
@pytest.mark.parametrize("rows", [1, 2, 70, 140])
@pytest.mark.parametrize("H,kv_rank,rot", [(3, 64, 16), (2, 256, 32)])
def test_one_matching_latent_just_inside_and_just_outside(H, kv_rank, rot, rows, window):
    """bfloat16: one cached row towers over all others for every query; it must carry exactly the rows that see it."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.attention import AttentionPlan

    D, page, n = kv_rank + rot, 16, 150 + rows
    for far in sorted({0, 15, 16, n - 1, n - 2, n - rows, n - rows - 1, n - 64, n - 65, max(0, n - window), max(0, n - window - 1),
                       max(0, n - rows - window), max(0, n - rows - window + 1)}):
        if far >= n:
            continue
        lat = torch.zeros(n, D)
        lat[:, 1] = 1.0
        lat[far] = 0.0
        lat[far, 2], lat[far, D - 1] = 1.0, 40.0           # the value it carries, and the match (in the rotated part)
        cache, table = _latent_cache([lat], page, D, far, torch.bfloat16)
        ctx = step_ctx([rows], list(range(n - rows, n)))
        q = torch.zeros(rows, H, D)
        q[:, :, D - 1] = 1.0
        out = torch.zeros(rows, H * kv_rank, device=DEV, dtype=torch.bfloat16)
        plan = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0, device=torch.device(DEV))
        ops.latent_attention(q.to(torch.bfloat16).to(DEV), cache, out, table, ctx, H, kv_rank, 1.0, window, plan=plan)
        got = out.float().view(rows, H, kv_rank)[:, :, 2].cpu()
        for i in range(rows):
            p = n - rows + i
            visible = far <= p and (not window or p - far < window)
            assert bool((got[i] > 0.9).all()) == visible and bool((got[i] < 0.1).all()) != visible, (far, p)


@pytest.mark.parametrize("M", [1, 7, 16, 17, 70, 129])
@pytest.mark.parametrize("H,N,K,rot,halves", [(3, 64, 64, 0, False), (5, 256, 64, 32, True), (2, 24, 8, 6, False), (4, 72, 200, 10, True), (1, 100, 40, 8, True)])
def test_product_per_head_on_the_tensor_cores_with_a_rotated_part_behind_it(H, N, K, rot, halves, M):
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(M + N)
    dt, dims = torch.bfloat16, rot // 4 * 2
    a_hs = -(-(K + rot) // 8) * 8 if not rot else K + rot
    if rot and a_hs % 8:
        rot = dims = 8
        a_hs = K + rot
    a = torch.randn(M, H * a_hs, device=DEV).to(dt)
    w = (torch.randn(H, N, K, device=DEV) / math.sqrt(K)).to(dt)
    pos = torch.randint(0, 5000, (M,), dtype=torch.int32, device=DEV)
    fr = 300.0 ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1))
    o_hs = N + rot
    for out_dt in (dt, torch.float32):
        out = torch.full((M, H * o_hs + 5), 7.0, device=DEV, dtype=out_dt)
        view = out[:, :H * o_hs] if not rot else torch.full((M, H * o_hs), 7.0, device=DEV, dtype=out_dt)
        ops.linear_heads(a, a_hs, w, view, o_hs, M, rot=(pos, fr.to(DEV), rot, dims, halves) if rot else None)
        x = a.double().cpu().view(M, H, a_hs)
        want = torch.einsum("mhk,hnk->mhn", x[..., :K], w.double().cpu())
        got = view.double().cpu().view(M, H, o_hs)
        tol = 1e-5 if out_dt == torch.float32 else 1e-2
        assert float(((got[..., :N] - want) / (want.abs() + 1)).abs().max()) < tol
        if rot:
            tail = x[..., K:K + rot]
            if halves:
                t = _turn_halves(tail, pos.cpu(), dims, fr, 1.0)
            else:
                t = tail.clone()
                ang = pos.cpu().double()[:, None] * fr
                c, sn = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
                u, v = tail[..., 0:dims:2], tail[..., 1:dims:2]
                t[..., 0:dims:2], t[..., 1:dims:2] = u * c - v * sn, v * c + u * sn
            assert float(((got[..., N:] - t) / (t.abs() + 1)).abs().max()) < tol
        else:
            assert float(out[:, H * o_hs:].float().min()) == 7.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rd,dims", [(10, 6), (16, 16), (8, 0)])
def test_latent_rotation_in_halves_with_a_wide_projection(rd, dims, dtype):
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(rd)
    dt, T, qr, kr, page, eps, base = DT[dtype], 6, 24, 20, 16, 1e-5, 77.0
    wide = torch.randn(T, qr + kr + rd + 40, device=DEV)
    proj = wide[:, 8:]
    wq, wkv = torch.rand(qr, device=DEV) + 0.5, torch.rand(kr, device=DEV) + 0.5
    fr = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / max(dims, 1))
    pos, ent = [5, 6, 7, 100, 15, 16], [0, 0, 0, 1, -1, 2]
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    table = i32([[3] + [-1] * 7, [-1] * 6 + [1, -1], [2, 0] + [-1] * 6])
    cache = torch.zeros(5, 1, 1, page, kr + rd, device=DEV, dtype=dt)
    cq, status = torch.zeros(T, qr, device=DEV, dtype=dt), torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.latent_prep(proj, qr, kr, rd, dims, fr.to(DEV), wq, wkv, eps, cq, cache, table, i32(ent), i32(pos), T, status, halves=True)
    s = proj.double().cpu()
    rms = lambda v, w: v / torch.sqrt((v ** 2).mean(-1, keepdim=True) + eps) * w.double().cpu()
    tol = 1e-5 if dtype == "float32" else 0.03
    assert int(status) == 0 and float((cq.double().cpu() - rms(s[:, :qr], wq)).abs().max()) < tol
    c = rms(s[:, qr:qr + kr], wkv)
    k_rot = _turn_halves(s[:, None, qr + kr:qr + kr + rd], torch.tensor(pos), dims, fr, 1.0)[:, 0]
    for t, (pg, slot) in {0: (3, 5), 1: (3, 6), 2: (3, 7), 3: (1, 100 % 16), 5: (0, 0)}.items():
        assert float((cache[pg, 0, 0, slot].double().cpu() - torch.cat([c[t], k_rot[t]])).abs().max()) < tol, t
    H, nope = 3, 4
    q = torch.randn(T, H * (nope + rd), device=DEV).to(dt)
    full = torch.zeros(T, H, kr + rd, device=DEV)
    ops.rope_heads(q, nope, rd, dims, fr.to(DEV), i32(pos), full, kr, H, T, halves=True)
    want = _turn_halves(q.double().cpu().view(T, H, nope + rd)[..., nope:], torch.tensor(pos), dims, fr, 1.0)
    assert float((full[..., kr:].double().cpu() - want).abs().max()) < 1e-5 and not full[..., :kr].any()


# =============================================================================== models through the step function
class Harness:
    def __init__(self, cfg, tmp_path, dtype, max_tokens=512, slots=4, page=16, max_rows=256, seed=1, sharpen=3.0,
                 long_memory=False):
        from nanoinfer_b200 import load_model
        from nanoinfer_b200.cache import CacheManager
        from nanoinfer_b200.engine import ModelRunner
        from plain_dedunex import PlainDedunex

        self.dir = write_model(cfg, str(tmp_path), DT[dtype], seed=seed, sharpen=sharpen, long_memory=long_memory)
        self.plain = PlainDedunex(self.dir)
        self.model = load_model(self.dir, DT[dtype], DEV)
        self.cache = CacheManager(self.model.kv_needs(), self.model.state_needs(), max_tokens=max_tokens,
                                  max_requests=slots, page_size=page, dtype=DT[dtype], device=torch.device(DEV),
                                  max_positions=self.model.max_positions, padding=True)
        self.runner = ModelRunner(self.model, self.cache, max_rows=max_rows, max_entries=slots, check_status=True)
        self.dtype, self.vocab = dtype, cfg["vocab"]

    def alone(self, tokens, cuts):
        """One request cut into portions of the sizes in ``cuts`` (cycled), all logits back."""
        from nanoinfer_b200.engine import StepItem

        r, at, k, rows = self.cache.open_request(), 0, 0, []
        while at < len(tokens):
            n = min(cuts[k % len(cuts)], len(tokens) - at)
            rows.append(self.runner.step([StepItem(r, tokens[at:at + n], list(range(n)))]).clone())
            at, k = at + n, k + 1
        self.cache.close_request(r)
        return torch.cat(rows)

    def check(self, got, tokens, what=""):
        assert_close(row_errs(got, self.plain.logits(tokens)), self.dtype, what)


ONE_LAYER = {
    "two maps": [diff_layer()],
    "two maps, a feed-forward beside them": [diff_layer(mlp=dense())],
    "two maps, one key head, a window of 7, all of a map turned": [diff_layer(heads=3, kv_heads=1, dim=12, vdim=30, window=7, rot=12)],
    "two maps, every head its own keys, no cap, plain rotation": [diff_layer(heads=2, kv_heads=2, dim=32, vdim=64, softcap=0, scaling=None)],
    "two maps, all keys, nothing turned, values shorter than a key": [diff_layer(heads=4, kv_heads=1, dim=24, vdim=8, window=0, rot=0, diff=0.9)],
    "two maps, a window of one position": [diff_layer(window=1)],
    "two maps of odd sizes": [diff_layer(heads=2, kv_heads=1, dim=9, vdim=21, rot=6, mlp=dense(27))],
    "two maps of 100 and values of 200": [diff_layer(heads=2, kv_heads=1, dim=100, vdim=200, rot=64, mlp=dense())],
    "a latent": [latent_layer()],
    "a latent, a feed-forward beside it": [latent_layer(mlp=dense())],
    "a latent, one head, values wider than keys, nothing turned": [latent_layer(heads=1, dim=8, rot_dim=0, vdim=40, q_rank=12, kv_rank=24)],
    "a latent, many heads, sizes of no multiple of eight": [latent_layer(heads=11, dim=10, rot_dim=6, vdim=9, q_rank=13, kv_rank=19, mlp=dense(20))],
    "a latent of 256 and 32": [latent_layer(heads=5, dim=32, rot_dim=32, vdim=32, q_rank=48, kv_rank=256, mlp=dense())],
    "a recurrent unit": [gru_layer()],
    "a recurrent unit of an odd size, a feed-forward beside it": [gru_layer(width=37, mlp=dense(50))],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ONE_LAYER))
def test_each_mechanism_alone_as_a_one_layer_model(name, dtype, tmp_path):
    h = Harness(config(ONE_LAYER[name], vocab=150, width=48), tmp_path, dtype)
    t = toks(150, 75, 3)
    h.check(h.alone(t, [1000]), t, name)
    h.check(h.alone(t, [40, 1, 1, 2, 3, 1]), t, name + " in portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("what", ["one norm group", "eight norm groups", "odd sizes and a large eps", "no loop", "one pass", "four passes of all layers",
                                  "a loop of one layer behind others", "a loop that ends the stack"])
def test_the_parts_around_the_layers(what, dtype, tmp_path):
    layers = [gru_layer(mlp=dense()), diff_layer(mlp=dense()), latent_layer()]
    kw = {"one norm group": dict(groups=1, loop=(0, 2, 2)), "eight norm groups": dict(groups=8, loop=(1, 3, 2)),
          "odd sizes and a large eps": dict(vocab=131, width=45, groups=3, eps=3e-2, loop=(0, 3, 2)), "no loop": dict(),
          "one pass": dict(loop=(1, 2, 1)), "four passes of all layers": dict(loop=(0, 3, 4)),
          "a loop of one layer behind others": dict(loop=(2, 3, 3)), "a loop that ends the stack": dict(loop=(1, 3, 2))}[what]
    cfg = config(layers, **{**dict(vocab=90, width=40), **kw})
    if what == "one norm group":
        del cfg["norm"]["groups"]
    h = Harness(cfg, tmp_path, dtype)
    t = toks(cfg["vocab"], 50, 6)
    h.check(h.alone(t, [1000]), t, what)
    h.check(h.alone(t, [30, 1, 2]), t, what + " in portions")
    h.check(h.alone(t, [1]), t, what + " one by one")


FULL = [gru_layer(width=56, mlp=dense(40)), diff_layer(mlp=dense(64)), latent_layer(mlp=dense(24)),
        diff_layer(heads=2, kv_heads=1, dim=32, vdim=32, window=40, rot=16, softcap=0, diff=0.7, mlp=None),
        latent_layer(heads=5, dim=8, rot_dim=16, vdim=16, q_rank=24, kv_rank=40, mlp=None), gru_layer(width=24, mlp=None)]
LOOP = (1, 5, 2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_token_by_token_and_portions_agree(dtype, tmp_path):
    h = Harness(config(FULL, vocab=190, width=64, eps=1e-6, loop=LOOP), tmp_path, dtype)
    t = toks(190, 97, 5)
    whole = h.alone(t, [1000])
    h.check(whole, t, "whole")
    ways = {"one by one": [1], "portions of two": [2], "3 and 5": [3, 5], "17, 16, 1, 31": [17, 16, 1, 31],
            "most of it, then single tokens": [60] + [1] * 40}
    for what, cuts in ways.items():
        got = h.alone(t, cuts)
        h.check(got, t, what)
        if dtype == "float32":     # how the prompt was cut shows in rounding only
            assert rel_err(got, whole) < 2e-5, what
    assert h.runner.graph_replays > 50            # single tokens ran as replayed graphs, states and all
    assert h.cache.pages_used() == [0] * len(h.cache.groups)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_together_equal_each_alone_and_pages_and_slots_come_back(dtype, tmp_path):
    from nanoinfer_b200.engine import StepItem

    h = Harness(config(FULL, vocab=170, width=64, loop=LOOP), tmp_path, dtype, max_tokens=4 * 64, slots=3)
    lens = [3, 120, 41, 64, 17, 88, 1]
    prompts = [toks(170, n, 20 + i) for i, n in enumerate(lens)]
    cuts = [[3], [50, 1, 1, 30, 2], [1, 40], [16, 16, 1], [17], [2, 2, 2, 80, 1], [1]]
    waiting, live, got = list(range(len(lens))), {}, {i: [] for i in range(len(lens))}
    slot_users, page_users, tick = {}, {}, 0
    while waiting or live:
        while waiting and len(live) < 3:
            i = waiting.pop(0)
            live[i] = [h.cache.open_request(), 0, 0]
            slot_users.setdefault(live[i][0].slot, set()).add(i)
        items, meta = [], []
        for j, (i, (req, at, k)) in enumerate(list(live.items())):
            if (tick + j) % 4 == 3 and len(live) > 1:
                continue                                   # sits this step out and goes on later
            n = min(cuts[i][k % len(cuts[i])], lens[i] - at)
            if not h.cache.can_append([(it.request, len(it.tokens)) for it in items] + [(req, n)]):
                continue
            items.append(StepItem(req, prompts[i][at:at + n], list(range(n))))
            meta.append((i, n))
        tick += 1
        if not items:
            continue
        out = h.runner.step(items)
        row = 0
        for i, n in meta:
            got[i].append(out[row:row + n].clone())
            row += n
            live[i][1] += n
            live[i][2] += 1
            for g, blocks in enumerate(live[i][0].blocks):
                for p in blocks:
                    if p >= 0:
                        page_users.setdefault((g, p), set()).add(i)
            if live[i][1] == lens[i]:
                h.cache.close_request(live[i][0])
                del live[i]
        h.cache.check()
    for i, t in enumerate(prompts):
        h.check(torch.cat(got[i]), t, f"request {i}")
    assert max(len(u) for u in slot_users.values()) >= 2 and max(len(u) for u in page_users.values()) >= 2
    assert h.cache.pages_used() == [0] * len(h.cache.groups) and h.cache.slots.n_free == 3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_lengths_around_page_and_window_edges_and_the_first_tokens(dtype, tmp_path):
    layers = [diff_layer(window=16, mlp=None), gru_layer(), latent_layer(), diff_layer(heads=2, kv_heads=1, dim=16, vdim=16, window=17, mlp=None)]
    h = Harness(config(layers, vocab=120, width=40, loop=(0, 2, 2)), tmp_path, dtype, sharpen=5.0)
    for n in (1, 2, 3, 15, 16, 17, 18, 31, 32, 33, 34, 47, 48, 49, 51):
        t = toks(120, n + 3, n)
        h.check(h.alone(t, [n, 1, 1, 1]), t, f"{n} tokens, then three alone")
        h.check(h.alone(t, [1, 1, 1, n]), t, f"three alone, then {n}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_behind_windows_and_through_states(dtype, tmp_path):
    """330 positions decoded; the windowed layers' pages come back while the latent layer keeps its own."""
    from nanoinfer_b200.engine import StepItem

    layers = [gru_layer(mlp=dense()), diff_layer(window=40, mlp=dense()), latent_layer(), diff_layer(window=21, mlp=None)]
    h = Harness(config(layers, vocab=100, width=48, loop=(1, 3, 2)), tmp_path, dtype, max_tokens=384, slots=2)
    t = toks(100, 330, 9)
    r = h.cache.open_request()
    rows = [h.runner.step([StepItem(r, t[:5], list(range(5)))]).clone()]
    for p in range(5, len(t)):
        rows.append(h.runner.step([StepItem(r, t[p:p + 1], [0])]).clone())
    used = h.cache.pages_used()
    assert min(used) <= -(-40 // 16) + 1 and max(used) == -(-330 // 16)
    h.cache.close_request(r)
    h.check(torch.cat(rows), t, "330 positions")
    assert h.runner.graph_replays > 300


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_long_prompts_through_the_tiled_prompt_kernels(dtype, tmp_path):
    """Cached rows of 64 (the tcgen05 prompt kernel in bfloat16), of 128, 96 and 48 (the warp-MMA one) and of 160 (the
    general one), latents of the usual size, over prompts of several tiles of keys: windows that end in the middle of a
    tile and of a page, windows longer than the prompt; whole, in portions that start anywhere, and with the last tokens
    one by one."""
    layers = [diff_layer(heads=4, kv_heads=2, dim=32, vdim=64, window=150, rot=32, mlp=dense()),
              latent_layer(heads=6, dim=64, rot_dim=32, vdim=64, q_rank=64, kv_rank=256, mlp=dense()),
              diff_layer(heads=2, kv_heads=1, dim=64, vdim=128, window=129, rot=16, mlp=None),
              diff_layer(heads=3, kv_heads=3, dim=48, vdim=96, window=2000, rot=8, mlp=None),
              latent_layer(heads=3, dim=24, rot_dim=16, vdim=40, q_rank=40, kv_rank=96, mlp=None),
              diff_layer(heads=2, kv_heads=2, dim=20, vdim=160, window=64, rot=8, mlp=None), gru_layer(width=64)]
    h = Harness(config(layers, vocab=150, width=64), tmp_path, dtype, max_tokens=1216, slots=2, max_rows=640, seed=5)
    tokens = toks(150, 590, 77)
    h.check(h.alone(tokens, [590]), tokens, "whole")
    h.check(h.alone(tokens, [333, 2, 131, 100] + [1] * 24), tokens, "in portions")
    assert h.cache.pages_used() == [0] * len(h.cache.groups)


def test_a_token_far_back_shows_through_the_state_and_through_the_latents(tmp_path):
    """A recurrent unit whose gates let it remember for hundreds of tokens, and attention through a latent that sees all
    keys: two prompts that differ in their first twelve tokens only still differ 150 tokens on, and the engine follows
    the plain model in both.  A windowed layer alone must not see them."""
    for layers, shows in (([gru_layer(width=48)], True), ([latent_layer(heads=4)], True), ([diff_layer(window=20)], False)):
        cfg = config(layers, vocab=90, width=64)
        h = Harness(cfg, tmp_path, "float32", long_memory=True, sharpen=6.0)
        a = toks(90, 150, 4)
        b = [(v + 1) % 90 for v in a[:12]] + a[12:]
        la, lb = h.plain.logits(a)[-1], h.plain.logits(b)[-1]
        far = rel_err(la[None], lb[None])
        assert far > 5 * TOL["float32"] if shows else far == 0.0, (layers[0]["type"], far)
        for t in (a, b):
            h.check(h.alone(t, [120, 7, 1]), t)
        if not shows:
            ea, eb = (h.alone(t, [120, 7, 1])[-1] for t in (a, b))
            assert torch.equal(ea, eb)


def random_config(rnd):
    width = rnd.choice([32, 40, 64, 72, 96, 100])
    groups = rnd.choice([g for g in (1, 2, 4, 5, 8) if width % g == 0])
    layers = []
    for _ in range(rnd.randint(1, 5)):
        mlp = dense(rnd.choice([8, 20, 33, 64, 96])) if rnd.random() < 0.7 else None
        kind = rnd.random()
        if kind < 0.3:
            layers.append(gru_layer(width=rnd.choice([8, 24, 33, 64, 130]), mlp=mlp))
        elif kind < 0.6:
            r = rnd.choice([0, 4, 16, 32])
            layers.append(latent_layer(heads=rnd.choice([1, 2, 5, 8, 9]), dim=rnd.choice([4, 16, 24, 64]), rot_dim=r,
                                       vdim=rnd.choice([8, 20, 64]), q_rank=rnd.choice([8, 24, 40]), kv_rank=rnd.choice([16, 32, 72, 128]),
                                       scale=rnd.choice([None, 0.3]), base=rnd.choice([50.0, 1e4, 1e6]), mlp=mlp))
        else:
            g = rnd.choice([1, 2, 3])
            dim = rnd.choice([8, 16, 24, 32, 64])
            layers.append(diff_layer(heads=g * rnd.choice([1, 2, 3]), kv_heads=g, dim=dim, vdim=rnd.choice([8, 24, 2 * dim, 100]),
                                     scale=rnd.choice([None, 0.2]), softcap=rnd.choice([0, 5.0, 50.0]), diff=rnd.choice([0.2, 0.5, 0.8]),
                                     window=rnd.choice([0, 1, 5, 16, 31, 64, 300]), rot=rnd.choice([0, 2, dim // 2, dim]),
                                     base=rnd.choice([100.0, 10000.0, 1e6]),
                                     scaling=rnd.choice([None, (2.0, 64, 8.0, 1.0), (4.0, 1024, 32.0, 1.0), (8.0, 20, 2.0, 0.25)]), mlp=mlp))
    a = rnd.randrange(len(layers))
    loop = (a, rnd.randint(a + 1, len(layers)), rnd.randint(1, 3)) if rnd.random() < 0.7 else None
    return config(layers, vocab=rnd.choice([50, 131, 256]), width=width, groups=groups, eps=rnd.choice([1e-6, 1e-5, 1e-3]), loop=loop)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", range(14))
def test_random_configuration_cut_at_random(case, dtype, tmp_path):
    from nanoinfer_b200.engine import StepItem

    rnd = random.Random(7300 + case)
    cfg = random_config(rnd)
    page = rnd.choice([16, 32, 48])
    lens = [rnd.randint(1, 150) for _ in range(rnd.randint(2, 6))]
    pages_of = lambda n: -(-n // page)
    pages = max(max(pages_of(n) for n in lens) + 2, int(0.6 * sum(pages_of(n) for n in lens)))
    h = Harness(cfg, tmp_path, dtype, max_tokens=pages * page, slots=3, page=page, max_rows=rnd.choice([64, 160]),
                seed=case + 1, sharpen=rnd.choice([2.0, 4.0]))
    prompts = [[rnd.randrange(cfg["vocab"]) for _ in range(n)] for n in lens]
    pending, live, got = list(range(len(lens))), {}, {}
    while pending or live:
        while pending and len(live) < 3:
            live[pending.pop(0)] = [h.cache.open_request(), 0]
        items, meta, rows = [], [], 0
        for i, (req, at) in list(live.items()):
            if rnd.random() < 0.2 and len(live) > 1:
                continue
            n = min(lens[i] - at, rnd.choice([1, 1, 2, 3, 7, 16, 17, 33, 64, 100]), h.runner.max_rows - rows)
            if n <= 0 or not h.cache.can_append([(it.request, len(it.tokens)) for it in items] + [(req, n)]):
                continue
            places = sorted(rnd.sample(range(n), min(n, rnd.randint(0, 3))))
            items.append(StepItem(req, prompts[i][at:at + n], places))
            meta.append((i, at, n, places))
            rows += n
        if not items:
            # nothing fits beside what is held: the newest request gives way and starts again later
            i = max(live)
            h.cache.close_request(live.pop(i)[0])
            pending.insert(0, i)
            got = {k: v for k, v in got.items() if k[0] != i}
            continue
        out = h.runner.step(items)
        k = 0
        for i, at, n, places in meta:
            for j in places:
                got[(i, at + j)] = out[k].clone()
                k += 1
            live[i][1] = at + n
            if at + n == lens[i]:
                h.cache.close_request(live.pop(i)[0])
    h.cache.check()
    assert got and h.cache.pages_used() == [0] * len(h.cache.groups)
    want = [h.plain.logits(t) for t in prompts]
    keys = sorted(got)
    errs = row_errs(torch.stack([got[k] for k in keys]), torch.stack([want[i][p] for i, p in keys]))
    assert_close(errs, dtype, f"case {case} {json.dumps(cfg)} at (request, position) {keys}")


def test_vectors_ahead_of_runs_of_an_arrangement_that_does_not_add_them_itself(tmp_path):
    """The schedule's vectors belong to the model, not to one arrangement: a plain pre-norm stack with vectors equals the
    same stack whose residual stream is given them by hand."""
    from nanoinfer_b200.cache import CacheManager
    from nanoinfer_b200.engine import ModelRunner, StepItem
    from nanoinfer_b200.models.model import Model
    from nanoinfer_b200.models.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
    from nanoinfer_b200.parts.base import TensorRef
    from nanoinfer_b200.weights import random_tensors, write_safetensors
    from nanoinfer_b200.weights.loader import load_weights

    c = 48
    norm = lambda n: PartSpec("rmsnorm", dict(width=c, eps=1e-5), {"weight": TensorRef(n)})
    gru = PartSpec("min_gru", dict(width=c, inner=40), {k: TensorRef("m." + k) for k in
                                                         ("z_weight", "z_bias", "x_weight", "x_bias", "g_weight", "out_weight")})
    ff = PartSpec("gated_mlp", dict(width=c, inner=32), {k: TensorRef("f." + k) for k in ("gate_weight", "up_weight", "down_weight")})

    def spec(vectors):
        return ModelSpec(width=c, embedding=PartSpec("token_embedding", dict(vocab_size=60, width=c), {"table": TensorRef("embed")}),
                         position=None, layers=[LayerSpec("pre_norm", {"norm_1": norm("n1"), "mixer": gru, "norm_2": norm("n2"), "feed_forward": ff})],
                         schedule=[ScheduleEntry(0, add_vector=0 if vectors else None), ScheduleEntry(0, add_vector=1 if vectors else None)],
                         final_norm=norm("fn"), head=PartSpec("linear_head", dict(vocab_size=60, width=c), {"weight": TensorRef("head")}),
                         stream_vectors=PartSpec("stream_vector_table", dict(count=2, width=c), {"table": TensorRef("steps")}))
    outs = []
    for vectors in (True, False):
        model = Model(spec(vectors))
        tensors = {k: v * 10 for k, v in random_tensors(model, 3, 0.02).items()}
        write_safetensors(str(tmp_path / "model.safetensors"), tensors)
        load_weights(model, str(tmp_path), torch.float32, torch.device(DEV))
        if not vectors:
            blk, f, t = model.layers[0], model.layers[0].forward, iter((0, 1))
            def by_hand(x, ctx, *a):
                x[:ctx.n_rows] += tensors["steps"][next(t)].to(DEV)
                f(x, ctx, *a)
            blk.forward = by_hand
        cache = CacheManager(model.kv_needs(), model.state_needs(), max_tokens=64, max_requests=1, page_size=16, dtype=torch.float32,
                             device=torch.device(DEV))
        runner = ModelRunner(model, cache, max_rows=32, max_entries=1, use_graphs=False)
        outs.append(runner.step([StepItem(cache.open_request(), toks(60, 20, 1), list(range(20)))]).clone())
    assert rel_err(outs[0], outs[1]) < 1e-6 and float(outs[0].std()) > 0


def test_greedy_generation_through_the_engine_and_its_scheduler(tmp_path):
    import nanoinfer_b200 as nb
    from plain_dedunex import PlainDedunex

    cfg = config(FULL, vocab=130, width=64, loop=LOOP)
    d = write_model(cfg, str(tmp_path), torch.float32, seed=3)
    plain = PlainDedunex(d)
    prompts = [toks(130, n, 40 + n) for n in (1, 9, 30, 55, 17)]
    eng = nb.Engine(d, dtype="float32", max_tokens=3 * 128, max_batch=3, max_rows=64)
    outs = eng.generate(prompts, nb.SamplingParams(max_new_tokens=20))
    for p, o in zip(prompts, outs):
        assert o == plain.greedy(p, 20)
    assert eng.runner.graph_replays > 0 and eng.cache.pages_used() == [0] * len(eng.cache.groups)


def test_trace_replay_of_a_model_folder(tmp_path):
    from plain_dedunex import PlainDedunex
    from trace_util import TraceSession

    cfg = config(FULL[:5], vocab=110, width=48, loop=(0, 3, 2))
    d = write_model(cfg, str(tmp_path / "m"), torch.float32, seed=8)
    plain = PlainDedunex(d)
    reqs = {f"r{i}": toks(110, n, 60 + i) for i, n in enumerate((50, 3, 64, 20, 33, 9))}
    s = TraceSession(d, "float32", tmp_path / "out", 4 * 64, 110)
    order, live, at = list(reqs), [], {r: 0 for r in reqs}
    k = 0
    while order or live:
        while order and len(live) < 4:
            live.append(order.pop(0))
        entries, ended = [], []
        for r in list(live):
            n = min([7, 1, 20, 2][k % 4], len(reqs[r]) - at[r])
            k += 1
            entries.append((r, reqs[r][at[r]:at[r] + n], range(n)))
            at[r] += n
            if at[r] == len(reqs[r]):
                ended.append(r)
                live.remove(r)
        s.step(entries, end=ended)
    s.close()
    for r, t in reqs.items():
        assert rel_err(s.stacked(r, len(t)), plain.logits(t)) <= TOL["float32"], r


def test_command_line_writes_a_folder_generates_from_it_and_profiles(tmp_path, capsys):
    from nanoinfer_b200 import cli
    from plain_dedunex import PlainDedunex

    d = str(tmp_path / "m")
    assert cli.main(["random-weights", "--config", "dedunex-tiny", "--seed", "6", "--out", d, "--dtype", "float32"]) == 0
    capsys.readouterr()
    prompt = toks(512, 12, 77)
    assert cli.main(["--weights", d, "generate", "--dtype", "float32", "--prompt-ids", ",".join(map(str, prompt)),
                     "--tokens", "10", "--temperature", "0.0", "--profile"]) == 0
    captured = capsys.readouterr()
    printed = [int(t) for t in captured.out.split()]
    assert printed == PlainDedunex(d).greedy(prompt, 10)
    assert "min_gru" in captured.err and "attn" in captured.err and "diff_combine" in captured.err

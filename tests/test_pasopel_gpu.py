"""Pasopel on the GPU: every new kernel and every kernel option alone against plain torch in float64, every mechanism alone
as a one-layer model, and whole models through the step function, cut into steps every way, against the plain implementation
(tests/plain_pasopel.py).  Test weights are made so that faults show (pasopel_util.write_model); where random values would
still hide one (a key at the edge of a window, a block that is just seen or not yet), the test builds queries and keys by
hand."""
import json
import math
import random

import pytest
import torch

from pasopel_util import TOL, assert_close_where_routing_is_clear, config, dense, latent_layer, moe, pooled_layer, rel_err, row_errs, write_model
from test_dedunex_gpu import _latent_cache
from test_mulavik_gpu import step_ctx, toks

pytestmark = pytest.mark.gpu

DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
DEV = "cuda"


def blocks_seen(p, window, pool):
    return max(0, p - window + 1) // pool if pool and window else 0


# =============================================================================== kernels alone
def _cache_with_pooled_rows(dt, G, hd, page, ks, vs, window, pool, first_rows, seed):
    """Pages of positions and of pooled rows in a scrambled order, one block table row an entry (pooled pages from column
    ``at`` on); what nobody holds is large; pages wholly behind every later query's window are gone.  ks, vs: [n, G, hd]."""
    g = torch.Generator().manual_seed(seed)
    nb = [-(-len(k) // page) for k in ks]
    npool = [max(1, -(-(len(k) // pool) // page)) if pool else 0 for k in ks]
    at = max(nb) + 1
    ids = torch.randperm(sum(nb) + sum(npool) + 3, generator=g).tolist()
    table = torch.full((len(ks), at + max(npool) + 1), -1, dtype=torch.int32)
    cache = torch.full((len(ids), 2, G, page, hd), 5.0)
    for e, (k, v) in enumerate(zip(ks, vs)):
        behind = max(0, first_rows[e] - window + 1) if window else 0
        for b in range(nb[e]):
            pg, c = ids.pop(), min(page, len(k) - b * page)
            if (b + 1) * page <= behind:
                continue
            table[e, b] = pg
            cache[pg, 0, :, :c] = k[b * page:b * page + c].transpose(0, 1)
            cache[pg, 1, :, :c] = v[b * page:b * page + c].transpose(0, 1)
        for b in range(npool[e]):
            table[e, at + b] = ids.pop()
        for b in range(len(k) // pool if pool else 0):
            pg = int(table[e, at + b // page])
            cache[pg, 0, :, b % page] = k[b * pool:(b + 1) * pool].double().mean(0).to(dt).float()
            cache[pg, 1, :, b % page] = v[b * pool:(b + 1) * pool].double().mean(0).to(dt).float()
    return cache.to(dt).to(DEV), table.to(DEV), at


def _pooled_reference(q, k, v, scale, positions, window, pool, sinks, dt):
    """q [n, H, d]; k, v [m, G, d] as the cache holds them; blocks' means rounded as the cache rounds them."""
    H, G = q.shape[1], k.shape[1]
    out = torch.zeros(len(positions), H, v.shape[2], dtype=torch.float64)
    nb = k.shape[0] // pool if pool else 0
    mean = lambda x: x[:nb * pool].double().view(nb, pool, *x.shape[1:]).mean(1).to(dt).double() if nb else x[:0].double()
    pk, pv = mean(k), mean(v)
    for i, p in enumerate(positions):
        lo = max(0, p - window + 1) if window else 0
        n = blocks_seen(p, window, pool)
        kk, vv = torch.cat([pk[:n], k[lo:p + 1].double()]), torch.cat([pv[:n], v[lo:p + 1].double()])
        for h in range(H):
            s = (kk[:, h // (H // G)] @ q[i, h].double()) * scale
            top = s.max() if sinks is None else torch.maximum(s.max(), sinks[h].double())
            e = torch.exp(s - top)
            den = e.sum() + (torch.exp(sinks[h].double() - top) if sinks is not None else 0.0)
            out[i, h] = (e[:, None] * vv[:, h // (H // G)]).sum(0) / den
    return out


POOLED_CASES = [(4, 2, 16, 16, 16), (6, 1, 48, 44, 16), (3, 3, 32, 32, 32), (12, 4, 64, 64, 16), (2, 1, 128, 120, 48), (20, 1, 64, 64, 16),
                (2, 2, 208, 200, 16), (4, 1, 256, 256, 16), (4, 2, 64, 64, 8)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window,pool", [(40, 8), (64, 16), (1, 1), (23, 5), (130, 3), (16, 40), (50, 0), (0, 0)])
@pytest.mark.parametrize("H,G,hd,dim,page", POOLED_CASES)
def test_window_and_pooled_blocks_in_one_softmax(H, G, hd, dim, page, window, pool, dtype):
    """Portions that start anywhere beside single tokens, portions alone, single tokens alone (their keys in one to many
    pieces), with sinks and a gate per element, with the pages behind the window gone: the tcgen05 and the warp-MMA kernels in
    bfloat16, the streaming and the general ones in float32 and for pages of 8."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.attention import AttentionPlan

    dt, scale = DT[dtype], 1.7 / math.sqrt(dim)
    for lengths, q_rows in (([200, 77, 301, 40, 16], [130, 1, 190, 3, 16]), ([300, 1, 77, 64], [1, 1, 1, 1]), ([129, 2, 128], [129, 2, 127])):
        g = torch.Generator().manual_seed(H + hd + len(lengths))
        pad = lambda x: torch.nn.functional.pad(x, (0, hd - dim))
        ks = [pad(torch.randn(n, G, dim, generator=g)).to(dt).float() for n in lengths]
        vs = [pad(torch.randn(n, G, dim, generator=g)).to(dt).float() for n in lengths]
        cache, table, at = _cache_with_pooled_rows(dt, G, hd, page, ks, vs, window, pool, [n - r for n, r in zip(lengths, q_rows)], H)
        positions = [p for n, r in zip(lengths, q_rows) for p in range(n - r, n)]
        n_pad = 3 if len(lengths) == 5 else 0
        ctx, T = step_ctx(q_rows, positions, n_pad=n_pad), len(positions)
        q = pad(torch.randn(T + n_pad, H, dim, generator=g)).to(dt)
        gate, sinks = torch.randn(T + n_pad, H * dim + 7, generator=g) * 2, torch.randn(H, generator=g) * 2
        out = torch.full((T + n_pad, H * hd + 8), 7.0, device=DEV, dtype=dt)
        plan = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0, device=torch.device(DEV))
        extras = ops.AttnExtras(sinks=sinks.to(DEV), gate=gate.to(DEV)[:, 3:3 + H * dim], gate_dim=dim, pool=pool,
                                pool_table=table[:, at:] if pool else None)
        ops.pooled_attention(q.view(-1, H * hd).to(DEV), cache, out[:, :H * hd], table, ctx, H, dim, scale, window, plan, extras)
        assert int(ctx.status.item()) == 0
        row, want = 0, []
        for e, (n, r) in enumerate(zip(lengths, q_rows)):
            o = _pooled_reference(q[row:row + r], ks[e], vs[e], scale, range(n - r, n), window, pool, sinks, dt)
            o[:, :, :dim] *= torch.sigmoid(gate[row:row + r, 3:3 + H * dim].double()).view(r, H, dim)
            want.append(o)
            row += r
        err = (out[:T, :H * hd].double().cpu() - torch.cat(want).reshape(T, -1)).abs()
        assert float(err.max()) < (2e-5 if dtype == "float32" else 4e-2), (lengths, float(err.max()), int(err.max(1).values.argmax()))
        assert float(out[:, H * hd:].float().min()) == 7.0 and float(out[T:].float().min() if n_pad else 7.0) == 7.0


@pytest.mark.parametrize("pieces", [1, 2, 4, 8, 16])
def test_single_tokens_whose_keys_are_cut_into_pieces_across_the_window(pieces):
    """bfloat16: the pieces of a row's keys begin among the pooled rows and end among the tokens."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.attention import AttentionPlan

    dt, H, G, hd, page, window, pool, n = torch.bfloat16, 10, 2, 32, 16, 70, 4, [900, 71, 3, 500]
    g = torch.Generator().manual_seed(pieces)
    ks, vs = ([torch.randn(m, G, hd, generator=g).to(dt).float() for m in n] for _ in range(2))
    cache, table, at = _cache_with_pooled_rows(dt, G, hd, page, ks, vs, window, pool, [m - 1 for m in n], 3)
    ctx = step_ctx([1] * 4, [m - 1 for m in n])
    q, sinks = torch.randn(4, H, hd, generator=g).to(dt), torch.randn(H, generator=g)
    out = torch.zeros(4, H * hd, device=DEV, dtype=dt)
    plan = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0, device=torch.device(DEV))
    assert ops.attention_group_mma(q.view(4, -1).to(DEV), cache, out, hd, table, ctx, plan, H, 0.3, window, hd, hd, n_splits=pieces,
                                   sinks=sinks.to(DEV), pool=pool, pool_table=table[:, at:])
    for e, m in enumerate(n):
        want = _pooled_reference(q[e:e + 1], ks[e], vs[e], 0.3, [m - 1], window, pool, sinks, dt)
        assert float((out[e].double().cpu() - want.reshape(-1)).abs().max()) < 2e-2, e


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [1, 2, 40, 150])
@pytest.mark.parametrize("window,pool", [(16, 4), (23, 5), (64, 16), (1, 3), (100, 64)])
def test_one_matching_key_or_block_just_inside_and_just_outside(window, pool, rows, dtype):
    """One cached row, of a position or of a block, towers over all others for every query; it must carry exactly the rows
    that see it: as a token inside the window, as a block behind it, and not at all in between."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.attention import AttentionPlan

    dt, H, hd, page, n = DT[dtype], 3, 64, 16, 220 + rows
    plain = [("token", j) for j in sorted({0, 15, 16, n - 1, n - 2, n - rows, n - rows - 1, n - window, n - window - 1, n - rows - window,
                                           n - rows - window + 1, n - 64, n - 65}) if 0 <= j < n]
    edge = [blocks_seen(p, window, pool) for p in (n - 1, n - rows)]
    plain += [("block", b) for b in sorted({0, 1, 15, 16, *[x + d for x in edge for d in (-2, -1, 0, 1)]}) if 0 <= b < n // pool]
    for kind, at_row in plain:
        k, v = torch.zeros(n, 1, hd), torch.zeros(n, 1, hd)
        cache, table, at = _cache_with_pooled_rows(dt, 1, hd, page, [k], [v], window, pool, [n - rows], at_row)
        tab = table.cpu()
        pg = int(tab[0, (at_row if kind == "token" else at * page + at_row) // page]) if kind == "token" else int(tab[0, at + at_row // page])
        if pg < 0:
            continue                                             # (a token whose page is gone)
        cache[pg, 0, 0, at_row % page, 5], cache[pg, 1, 0, at_row % page, 2] = 40.0, 1.0
        ctx = step_ctx([rows], list(range(n - rows, n)))
        q = torch.zeros(rows, H, hd)
        q[:, :, 5] = 1.0
        out = torch.zeros(rows, H * hd, device=DEV, dtype=dt)
        plan = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0, device=torch.device(DEV))
        ops.pooled_attention(q.view(rows, -1).to(dt).to(DEV), cache, out, table, ctx, H, hd, 1.0, window, plan,
                             ops.AttnExtras(pool=pool, pool_table=table[:, at:]))
        got = out.float().view(rows, H, hd)[:, :, 2].cpu()
        assert int(ctx.status.item()) == 0
        for i in range(rows):
            p = n - rows + i
            visible = 0 <= p - at_row < window if kind == "token" else at_row < blocks_seen(p, window, pool)
            assert bool((got[i] > 0.9).all()) == visible and bool((got[i] < 0.1).all()) != visible, (kind, at_row, p)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,dim,taps,pool,norm,page", [(4, 2, 16, 3, 8, True, 16), (6, 1, 44, 4, 5, True, 16), (3, 3, 32, 1, 1, True, 32),
                                                         (9, 3, 100, 2, 16, True, 16), (2, 1, 200, 3, 40, False, 48), (1, 1, 8, 5, 0, True, 16)])
def test_convolution_norm_cache_write_and_pooled_rows(H, G, dim, taps, pool, norm, page, dtype):
    """One request in portions cut anywhere (single rows shift the state themselves) beside another and padding: queries,
    cached keys and values and pooled rows against the formula; the state carries across every cut, also portions shorter
    than the taps; what was pooled does not depend on the cut."""
    from nanoinfer_b200.kernels import ops

    dt, hd, n = DT[dtype], -(-dim // 16) * 16, 70
    chans, eps = (H + G) * dim, 3e-5
    g = torch.Generator().manual_seed(dim + taps)
    u = [torch.randn(n, chans, generator=g) for _ in range(2)]
    w = torch.randn(chans, taps, generator=g)
    tol = 3e-6 if dtype == "float32" else 2e-2

    def formula(x):
        xx = torch.cat([torch.zeros(taps - 1, chans), x]).double()
        y = sum(w[:, j].double() * xx[j:j + n] for j in range(taps)).view(n, H + G, dim)
        return y, y / torch.sqrt((y ** 2).mean(-1, keepdim=True) + eps) if norm else y
    pools = []
    for cuts in ([70], [1] * 70, [5, 1, 1, 2, 30, 1, 16, 14], [2] * 35):
        nblk, npool = -(-n // page), max(1, -(-(n // pool) // page)) if pool else 0
        ids = torch.randperm(2 * (nblk + npool) + 2, generator=torch.Generator().manual_seed(1)).tolist()
        table = torch.tensor([[ids.pop() for _ in range(nblk + npool)] for _ in range(2)], dtype=torch.int32, device=DEV)
        cache = torch.full((2 * (nblk + npool) + 2, 2, G, page, hd), 9.0, device=DEV, dtype=dt)
        state = torch.zeros(4, max(taps - 1, 1) * chans + 4, device=DEV)
        at = 0
        for c in cuts:
            # (the other request runs along where the cuts are all alike, and in the first step otherwise)
            entries = [0, 1] if at == 0 or len(set(cuts)) == 1 else [0]
            ctx = step_ctx([c] * len(entries), list(range(at, at + c)) * len(entries), slots=[2, 0][:len(entries)], n_pad=0 if c == 1 else 2)
            proj = torch.full((ctx.n_rows, chans + 11), 3.0, device=DEV)
            for k, e in enumerate(entries):
                proj[k * c:(k + 1) * c, :chans] = u[e][at:at + c].to(DEV)
            q = torch.full((ctx.n_rows, H * hd), 9.0, device=DEV, dtype=dt)
            ops.conv_pool_append(proj, taps, w.t().contiguous().to(DEV), state if taps > 1 else None, H, G, dim, norm, eps, pool,
                                 ctx, q, cache, table, table[:, nblk:] if pool else None)
            assert int(ctx.status.item()) == 0
            for k, e in enumerate(entries):
                want = formula(u[e])[1][at:at + c, :H]
                got = q[k * c:(k + 1) * c].double().cpu().view(c, H, hd)
                assert float(((got[..., :dim] - want) / (want.abs() + 1)).abs().max()) < tol, (cuts, at)
                assert not got[..., dim:].any()
            at += c
        y, nk = formula(u[0])
        flat = lambda plane: torch.cat([cache[int(p), plane].transpose(0, 1) for p in table[0, :nblk]])[:n].double().cpu()
        for plane, want in ((0, nk[:, H:]), (1, y[:, H:])):
            got = flat(plane)
            assert float(((got[..., :dim] - want) / (want.abs() + 1)).abs().max()) < tol and not got[..., dim:].any()
        if pool:
            rows = torch.cat([cache[int(p)].permute(2, 0, 1, 3) for p in table[0, nblk:]])[:n // pool].double().cpu()
            means = torch.stack([torch.stack([flat(plane)[b * pool:(b + 1) * pool].mean(0) for plane in (0, 1)]) for b in range(n // pool)])
            assert float((rows - means).abs().max()) < (1e-6 if dtype == "float32" else 2e-2)
            pools.append(rows)
    assert all(torch.equal(p, pools[0]) for p in pools)          # to the bit


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window", [0, 70, 1])
@pytest.mark.parametrize("H,kv_rank,rot,page", [(3, 32, 8, 16), (12, 128, 32, 48), (4, 256, 32, 16), (2, 512, 64, 16), (17, 96, 24, 16), (3, 336, 48, 16)])
def test_latent_attention_with_learned_sinks(H, kv_rank, rot, page, window, dtype):
    """Every kernel of the latent attention (tcgen05, warp-MMA, the general one whole and in pieces)."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.attention import AttentionPlan

    dt, D, scale = DT[dtype], kv_rank + rot, 1.5 / math.sqrt(kv_rank)
    for lengths, q_rows in (([200, 77, 301, 16], [130, 1, 260, 16]), ([300, 1, 77], [1, 1, 1])):
        g = torch.Generator().manual_seed(H + kv_rank)
        lats = [torch.randn(n, D, generator=g).to(dt).float() for n in lengths]
        cache, table = _latent_cache(lats, page, D, H, dt)
        positions = [p for n, r in zip(lengths, q_rows) for p in range(n - r, n)]
        ctx, T = step_ctx(q_rows, positions), len(positions)
        q, sinks = torch.randn(T, H, D, generator=g).to(dt), torch.randn(H, generator=g) * 2
        out = torch.zeros(T, H * kv_rank, device=DEV, dtype=dt)
        plan = AttentionPlan(ctx.host_entry_start, ctx.host_entry_pos0, device=torch.device(DEV))
        ops.latent_attention(q.to(DEV), cache, out, table, ctx, H, kv_rank, scale, window, plan=plan, sinks=sinks.to(DEV))
        assert int(ctx.status.item()) == 0
        row = 0
        for e, (n, r) in enumerate(zip(lengths, q_rows)):
            for i in range(r):
                p = n - r + i
                lo = max(0, p - window + 1) if window else 0
                kk = lats[e][lo:p + 1].double()
                s = torch.einsum("hd,jd->hj", q[row + i].double(), kk) * scale
                ex = torch.exp(s)
                want = (ex @ kk[:, :kv_rank]) / (ex.sum(1) + torch.exp(sinks.double()))[:, None]
                err = float((out[row + i].double().cpu() - want.reshape(-1)).abs().max())
                assert err < (2e-5 if dtype == "float32" else 4e-2), (e, p, err)
            row += r


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,N,K,M", [(3, 64, 64, 7), (5, 24, 40, 70), (2, 100, 96, 17), (4, 9, 19, 1)])
def test_product_per_head_with_a_gate_per_element(H, N, K, M, dtype):
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(N)
    dt = DT[dtype]
    a, w = torch.randn(M, H * K, device=DEV).to(dt), (torch.randn(H, N, K, device=DEV) / math.sqrt(K)).to(dt)
    gate = torch.randn(M, H * N + 5, device=DEV) * 2
    out = torch.full((M, H * N + 3), 7.0, device=DEV, dtype=dt)
    ops.linear_heads(a, K, w, out[:, :H * N], N, M, gate=gate[:, 2:2 + H * N])
    want = torch.einsum("mhk,hnk->mhn", a.double().view(M, H, K), w.double()).reshape(M, -1) * torch.sigmoid(gate[:, 2:2 + H * N].double())
    assert float(((out[:, :H * N].double() - want) / (want.abs() + 1)).abs().max()) < (1e-5 if dtype == "float32" else 1e-2)
    assert float(out[:, H * N:].float().min()) == 7.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,top,C", [(5, 2, 72), (16, 4, 1000), (40, 1, 45), (3, 3, 768), (7, 2, 2056)])
def test_routing_by_biased_logits(E, top, C, dtype):
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(E)
    dt, T = DT[dtype], 30
    h, w, b = torch.randn(T, C, device=DEV).to(dt), (torch.randn(E, C, device=DEV) / C ** 0.5).to(dt), torch.randn(E, device=DEV)
    ids, weights = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV)
    ops.moe_route(h, w, T, top, True, ids, weights, logit_bias=b)
    z = h.double() @ w.double().T + b.double()
    best = torch.topk(z, top, dim=1)
    assert torch.equal(ids.long(), best.indices)
    assert float((weights.double() - torch.softmax(best.values, 1)).abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("M", [1, 8, 9, 16, 40, 130])
@pytest.mark.parametrize("N,K", [(96, 48), (200, 768), (64, 1600), (33, 100)])
def test_product_of_an_rms_norm_of_the_stream(N, K, M, dtype):
    """The norm folded into the product of few rows (no shift, nothing taken off), or run ahead of it; rows picked."""
    from nanoinfer_b200.kernels import ops
    from nanoinfer_b200.parts.base import Workspace

    torch.manual_seed(N + M)
    dt, eps = DT[dtype], 1e-4
    x, g = torch.randn(M + 5, K, device=DEV) + 0.7, torch.rand(K, device=DEV) + 0.5
    w, b = (torch.randn(N, K, device=DEV) / K ** 0.5).to(dt), torch.randn(N, device=DEV)
    rows = torch.randperm(M + 5, device=DEV)[:M].to(torch.int32)
    for r in (None, rows):
        norm = ops.NormInput(x, g, None, eps, Workspace(torch.device(DEV)), dt, rows=r)
        out = torch.full((M, N), 7.0, device=DEV)
        ops.linear(None, w, b, out, M, norm=norm)
        xr = (x[:M] if r is None else x[r.long()]).double()
        y = (xr / torch.sqrt((xr ** 2).mean(-1, keepdim=True) + eps) * g.double()).to(dt).double()
        want = y @ w.double().T + b.double()
        assert float((out.double() - want).abs().max()) < (1e-5 if dtype == "float32" else 3e-2)


@pytest.mark.parametrize("M", [17, 128, 130, 700])
@pytest.mark.parametrize("S,N,F", [(3, 64, 64), (8, 768, 128), (5, 72, 192), (16, 200, 64), (2, 1600, 1600), (1, 48, 320)])
def test_one_product_over_stacked_matrices(S, N, F, M):
    """The K of one product walks matrices that lie one after another (tcgen05, TMA coordinates by segment), stored and added."""
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(M + N)
    a = torch.randn(M + 3, S * F, device=DEV).to(torch.bfloat16)
    w = (torch.randn(S, N, F, device=DEV) / (S * F) ** 0.5).to(torch.bfloat16)
    want = sum(a[:M, s * F:(s + 1) * F].double() @ w[s].double().T for s in range(S))
    x0 = torch.randn(M + 3, N, device=DEV)
    for residual in (True, False):
        x = x0.clone()
        assert ops.linear_segments(a, w, x, M, residual=residual)
        assert int(ops.status_word()) == 0
        ref = want + (x0[:M].double() if residual else 0.0)
        assert float((x[:M].double() - ref).abs().max()) < 1e-3 and torch.equal(x[M:], x0[M:])


@pytest.mark.parametrize("F", [64, 24, 30])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gated_experts_all_at_once(F, dtype):
    """A step of many rows: all experts through the engine's products, what a row did not choose zeroed and not read (what
    lies there is not a number), by the four-a-thread kernel and the plain one."""
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(F)
    dt, T, E, top = DT[dtype], 21, 6, 2
    pre = torch.randn(T, E * 2 * F, device=DEV)
    ids = torch.stack([torch.randperm(E, device=DEV)[:top] for _ in range(T)]).to(torch.int32)
    weights = torch.rand(T, top, device=DEV)
    want = torch.zeros(T, E, F, dtype=torch.float64, device=DEV)
    p = pre.double().view(T, E, F, 2)
    chosen = torch.zeros(T, E, dtype=torch.bool, device=DEV)
    for k in range(top):
        r = torch.arange(T, device=DEV)
        g, u = p[r, ids[:, k].long(), :, 0], p[r, ids[:, k].long(), :, 1]
        want[r, ids[:, k].long()] = weights[:, k:k + 1].double() * g * torch.sigmoid(g) * u
        chosen[r, ids[:, k].long()] = True
    pre.view(T, E, 2 * F)[~chosen] = float("nan")
    out = torch.full((T, E * F), 7.0, device=DEV, dtype=dt)
    ops.moe_gate_scale(pre, out, ids, weights, T, E, F, top, ops.ACT_SILU, False)
    assert float((out.double() - want.view(T, -1)).abs().max()) < (1e-5 if dtype == "float32" else 3e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,groups", [(40, 1), (264, 2), (30, 3), (1536, 1), (768, 1), (2048, 1)])
def test_norm_with_rows_and_a_vector_added_first(C, groups, dtype):
    from nanoinfer_b200.kernels import ops

    torch.manual_seed(C)
    T, R, eps = 9, 12, 3e-5
    x0, rows, add, w = torch.randn(R, C, device=DEV), torch.randn(R, C, device=DEV), torch.randn(C, device=DEV), torch.rand(C, device=DEV) + 0.5
    for a in (add, None):
        want = x0[:T] + rows[:T] + (a if a is not None else 0.0)
        x, out = x0.clone(), torch.zeros(R, C, device=DEV, dtype=DT[dtype])
        ops.group_norm(x, w, groups, eps, out, T, add=a, add_rows=rows)
        p = want.double().view(T, groups, -1)
        ref = (p / torch.sqrt((p ** 2).mean(-1, keepdim=True) + eps)).view(T, C) * w.double()
        assert float((x[:T] - want).abs().max()) < 1e-6 and torch.equal(x[T:], x0[T:])
        assert float(((out[:T].double() - ref) / (ref.abs() + 1)).abs().max()) < (3e-6 if dtype == "float32" else 1e-2)
        x = x0.clone()
        ops.group_norm(x, None, 1, 0.0, None, T, add=a, add_rows=rows)       # the sum alone
        assert float((x[:T] - want).abs().max()) < 1e-6 and torch.equal(x[T:], x0[T:])


# =============================================================================== models through the step function
class Harness:
    def __init__(self, cfg, tmp_path, dtype, max_tokens=512, slots=4, page=16, max_rows=256, seed=1, sharpen=3.0):
        from nanoinfer_b200 import load_model
        from nanoinfer_b200.cache import CacheManager
        from nanoinfer_b200.engine import ModelRunner
        from plain_pasopel import PlainPasopel

        self.dir = write_model(cfg, str(tmp_path), DT[dtype], seed=seed, sharpen=sharpen)
        self.plain = PlainPasopel(self.dir)
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
        assert_close_where_routing_is_clear(row_errs(got, self.plain.logits(tokens)), self.plain.margins(tokens), self.dtype, what)


ONE_LAYER = {
    "a window and pooled blocks": [pooled_layer()],
    "blocks longer than the window": [pooled_layer(window=5, pool=12)],
    "blocks of one token, a window of one": [pooled_layer(window=1, pool=1)],
    "one key head, a window of no multiple of its blocks, four taps": [pooled_layer(heads=5, kv_heads=1, dim=24, conv=4, window=19, pool=7)],
    "every head its own keys, one tap, a dense feed-forward": [pooled_layer(heads=3, kv_heads=3, dim=32, conv=1, window=16, pool=16, mlp=dense())],
    "no convolution, all keys": [pooled_layer(conv=0, window=0, pool=0)],
    "a window without blocks": [pooled_layer(window=9, pool=0, conv=2)],
    "heads of an odd size": [pooled_layer(heads=4, kv_heads=2, dim=13, window=20, pool=4, mlp=dense(27))],
    "heads of 64": [pooled_layer(heads=6, kv_heads=2, dim=64, window=33, pool=8)],
    "heads of 136": [pooled_layer(heads=2, kv_heads=1, dim=136, window=30, pool=5)],
    "a latent behind a window": [latent_layer()],
    "a latent, one head, values wider than keys, nothing turned, all keys": [latent_layer(heads=1, dim=8, rot_dim=0, vdim=40, q_rank=12, kv_rank=24, window=0)],
    "a latent, many heads, sizes of no multiple of eight": [latent_layer(heads=11, dim=10, rot_dim=6, vdim=9, q_rank=13, kv_rank=19, window=7, mlp=dense(20))],
    "a latent of 256 and 32": [latent_layer(heads=5, dim=32, rot_dim=32, vdim=32, q_rank=48, kv_rank=256, window=50)],
    "experts, a shared one": [latent_layer(window=1, mlp=moe())],
    "experts, none shared, three of eleven": [pooled_layer(mlp=moe(11, 3, 20, 0))],
    "one expert of many": [pooled_layer(mlp=moe(24, 1, 33, 17))],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(ONE_LAYER))
def test_each_mechanism_alone_as_a_one_layer_model(name, dtype, tmp_path):
    h = Harness(config(ONE_LAYER[name], vocab=150, width=48), tmp_path, dtype)
    t = toks(150, 75, 3)
    h.check(h.alone(t, [1000]), t, name)
    h.check(h.alone(t, [40, 1, 1, 2, 3, 1]), t, name + " in portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("what", ["odd sizes and a large eps", "no loop, no cap", "one pass", "four passes of all layers",
                                  "a loop of one layer behind others", "a loop that ends the stack"])
def test_the_parts_around_the_layers(what, dtype, tmp_path):
    layers = [pooled_layer(mlp=dense()), latent_layer(mlp=moe()), pooled_layer(window=7, pool=3)]
    kw = {"odd sizes and a large eps": dict(vocab=131, width=45, eps=3e-2, loop=(0, 3, 2)), "no loop, no cap": dict(cap=0),
          "one pass": dict(loop=(1, 2, 1)), "four passes of all layers": dict(loop=(0, 3, 4)),
          "a loop of one layer behind others": dict(loop=(2, 3, 3)), "a loop that ends the stack": dict(loop=(1, 3, 2), cap=5.0)}[what]
    cfg = config(layers, **{**dict(vocab=90, width=40), **kw})
    h = Harness(cfg, tmp_path, dtype)
    t = toks(cfg["vocab"], 50, 6)
    h.check(h.alone(t, [1000]), t, what)
    h.check(h.alone(t, [30, 1, 2]), t, what + " in portions")
    h.check(h.alone(t, [1]), t, what + " one by one")


FULL = [pooled_layer(mlp=dense(64)), latent_layer(mlp=moe(7, 2, 24, 16)), pooled_layer(heads=3, kv_heads=1, dim=32, conv=4, window=18, pool=5, mlp=moe(4, 2, 32, 0)),
        latent_layer(heads=5, dim=8, rot_dim=16, vdim=16, q_rank=24, kv_rank=40, window=33), pooled_layer(heads=2, kv_heads=2, dim=48, window=40, pool=16, mlp=dense(24))]
LOOP = (1, 4, 2)


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
                for p in [*blocks, *live[i][0].pooled[g]]:
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
def test_batches_of_single_tokens_are_filled_up_with_rows_of_no_request(dtype, tmp_path):
    """More than eight single tokens: the step is padded with rows that point at the spare page and slot, also where every
    position ends a block."""
    from nanoinfer_b200.engine import StepItem

    h = Harness(config([pooled_layer(window=3, pool=1), pooled_layer(window=5, pool=2, mlp=dense())], vocab=80, width=40), tmp_path,
                dtype, max_tokens=512, slots=12)
    prompts = [toks(80, 24, i) for i in range(11)]
    reqs = [h.cache.open_request() for _ in prompts]
    got = [[] for _ in prompts]
    for at in range(24):
        out = h.runner.step([StepItem(r, [t[at]], [0]) for r, t in zip(reqs, prompts)])
        for i in range(len(prompts)):
            got[i].append(out[i].clone())
    assert h.runner.padded_steps > 0
    for t, g in zip(prompts, got):
        h.check(torch.stack(g), t)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_lengths_around_page_window_and_block_edges_and_the_first_tokens(dtype, tmp_path):
    layers = [pooled_layer(window=16, pool=16), latent_layer(window=17), pooled_layer(heads=2, kv_heads=1, window=17, pool=8, conv=2), pooled_layer(window=8, pool=3)]
    h = Harness(config(layers, vocab=120, width=40, loop=(0, 2, 2)), tmp_path, dtype, sharpen=5.0)
    for n in (1, 2, 3, 15, 16, 17, 18, 31, 32, 33, 34, 47, 48, 49, 51):
        t = toks(120, n + 3, n)
        h.check(h.alone(t, [n, 1, 1, 1]), t, f"{n} tokens, then three alone")
        h.check(h.alone(t, [1, 1, 1, n]), t, f"three alone, then {n}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_behind_windows(dtype, tmp_path):
    """330 positions decoded through a pool that holds 192: the positions' pages come back behind the windows, pooled rows
    stay, block tables grow."""
    from nanoinfer_b200.engine import StepItem

    layers = [pooled_layer(window=40, pool=4, mlp=dense()), latent_layer(window=30, mlp=moe()), pooled_layer(window=21, pool=9, mlp=None)]
    h = Harness(config(layers, vocab=100, width=48, loop=(1, 3, 2)), tmp_path, dtype, max_tokens=192, slots=2)
    t = toks(100, 330, 9)
    r = h.cache.open_request()
    rows = [h.runner.step([StepItem(r, t[:5], list(range(5)))]).clone()]
    for p in range(5, len(t)):
        rows.append(h.runner.step([StepItem(r, t[p:p + 1], [0])]).clone())
    assert [len(g) for g in r.pooled] == [-(-(330 // g.spec.pool) // 16) if g.spec.pool else 0 for g in h.cache.groups]
    assert max(sum(1 for p in b if p >= 0) for b in r.blocks) <= -(-40 // 16) + 1
    h.cache.close_request(r)
    h.check(torch.cat(rows), t, "330 positions")
    assert h.runner.graph_replays > 250


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_long_prompts_through_the_tiled_prompt_kernels(dtype, tmp_path):
    """Prompts of several tiles of keys and of pooled rows: heads of 48, 64, 128 and 160, windows and blocks that end in the
    middle of a tile and of a page; whole, in portions that start anywhere, and with the last tokens one by one."""
    layers = [pooled_layer(heads=4, kv_heads=2, dim=64, window=150, pool=2, mlp=dense()),
              latent_layer(heads=6, dim=64, rot_dim=32, vdim=64, q_rank=64, kv_rank=256, window=100, mlp=moe()),
              pooled_layer(heads=2, kv_heads=1, dim=128, window=129, pool=3, mlp=None),
              pooled_layer(heads=3, kv_heads=3, dim=40, window=64, pool=5, mlp=None), pooled_layer(heads=2, kv_heads=1, dim=160, window=20, pool=16, mlp=None)]
    h = Harness(config(layers, vocab=150, width=64), tmp_path, dtype, max_tokens=1216, slots=2, max_rows=640, seed=5)
    tokens = toks(150, 590, 77)
    h.check(h.alone(tokens, [590]), tokens, "whole")
    h.check(h.alone(tokens, [333, 2, 131, 100] + [1] * 24), tokens, "in portions")
    assert h.cache.pages_used() == [0] * len(h.cache.groups)


def test_a_token_far_back_shows_through_its_block_alone(tmp_path):
    """Two prompts that differ in their first twelve tokens only: 150 tokens on, the pooled blocks still tell them apart, a
    window without blocks does not."""
    for layer, shows in ((pooled_layer(window=20, pool=4), True), (pooled_layer(window=20, pool=0), False), (latent_layer(window=20), False)):
        h = Harness(config([layer], vocab=90, width=64), tmp_path, "float32", sharpen=6.0)
        a = toks(90, 150, 4)
        b = [(v + 1) % 90 for v in a[:12]] + a[12:]
        la, lb = h.plain.logits(a)[-1], h.plain.logits(b)[-1]
        far = rel_err(la[None], lb[None])
        assert far > 5 * TOL["float32"] if shows else far == 0.0, far
        for t in (a, b):
            h.check(h.alone(t, [120, 7, 1]), t)
        if not shows:
            ea, eb = (h.alone(t, [120, 7, 1])[-1] for t in (a, b))
            assert torch.equal(ea, eb)


def random_config(rnd):
    layers = []
    for _ in range(rnd.randint(1, 4)):
        kind = rnd.random()
        mlp = None if kind < 0.2 else dense(rnd.choice([8, 20, 33, 64, 96])) if kind < 0.5 else moe(
            *rnd.choice([(4, 1), (5, 3), (9, 2), (16, 2)]), rnd.choice([8, 24, 33]), rnd.choice([0, 16, 40]))
        if rnd.random() < 0.4:
            layers.append(latent_layer(heads=rnd.choice([1, 2, 5, 8, 9]), dim=rnd.choice([4, 16, 24, 64]), rot_dim=rnd.choice([0, 4, 16, 32]),
                                       vdim=rnd.choice([8, 20, 64]), q_rank=rnd.choice([8, 24, 40]), kv_rank=rnd.choice([16, 32, 72, 128]),
                                       scale=rnd.choice([None, 0.3]), base=rnd.choice([50.0, 1e4, 1e6]), window=rnd.choice([0, 1, 5, 16, 31, 64]), mlp=mlp))
        else:
            g = rnd.choice([1, 2, 3])
            layers.append(pooled_layer(heads=g * rnd.choice([1, 2, 3]), kv_heads=g, dim=rnd.choice([8, 16, 20, 32, 48, 64, 96]), conv=rnd.choice([0, 1, 2, 3, 4]),
                                       scale=rnd.choice([None, 0.2]), window=rnd.choice([1, 5, 16, 31, 64]), pool=rnd.choice([0, 1, 2, 5, 8, 16, 24]), mlp=mlp))
    a = rnd.randrange(len(layers))
    loop = (a, rnd.randint(a + 1, len(layers)), rnd.randint(1, 3)) if rnd.random() < 0.7 else None
    return config(layers, vocab=rnd.choice([50, 131, 256]), width=rnd.choice([32, 40, 64, 72, 96, 100]), eps=rnd.choice([1e-6, 1e-5, 1e-3]),
                  loop=loop, cap=rnd.choice([0, 8.0, 30.0]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", range(14))
def test_random_configuration_cut_at_random(case, dtype, tmp_path):
    from nanoinfer_b200.engine import StepItem

    rnd = random.Random(8100 + case)
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
    sure = [h.plain.margins(t) for t in prompts]
    assert_close_where_routing_is_clear(errs, torch.stack([sure[i][p] for i, p in keys]), dtype, f"case {case} {json.dumps(cfg)} at (request, position) {keys}")


def test_greedy_generation_through_the_engine_and_its_scheduler(tmp_path):
    import nanoinfer_b200 as nb
    from plain_pasopel import PlainPasopel

    cfg = config(FULL, vocab=130, width=64, loop=LOOP)
    d = write_model(cfg, str(tmp_path), torch.float32, seed=3)
    plain = PlainPasopel(d)
    prompts = [toks(130, n, 40 + n) for n in (1, 9, 30, 55, 17)]
    eng = nb.Engine(d, dtype="float32", max_tokens=3 * 128, max_batch=3, max_rows=64)
    outs = eng.generate(prompts, nb.SamplingParams(max_new_tokens=20))
    for p, o in zip(prompts, outs):
        assert o == plain.greedy(p, 20)
    assert eng.runner.graph_replays > 0 and eng.cache.pages_used() == [0] * len(eng.cache.groups)


def test_trace_replay_of_a_model_folder(tmp_path):
    from plain_pasopel import PlainPasopel
    from trace_util import TraceSession

    cfg = config(FULL, vocab=110, width=48, loop=(0, 3, 2))
    d = write_model(cfg, str(tmp_path / "m"), torch.float32, seed=8)
    plain = PlainPasopel(d)
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
    from plain_pasopel import PlainPasopel

    d = str(tmp_path / "m")
    assert cli.main(["random-weights", "--config", "pasopel-tiny", "--seed", "6", "--out", d, "--dtype", "float32"]) == 0
    capsys.readouterr()
    prompt = toks(512, 12, 77)
    assert cli.main(["--weights", d, "generate", "--dtype", "float32", "--prompt-ids", ",".join(map(str, prompt)),
                     "--tokens", "10", "--temperature", "0.0", "--profile"]) == 0
    captured = capsys.readouterr()
    printed = [int(t) for t in captured.out.split()]
    assert printed == PlainPasopel(d).greedy(prompt, 10)
    assert "norm_kv_write" in captured.err and "attn" in captured.err and "latent_attn" in captured.err

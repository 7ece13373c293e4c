"""Mixed stacks on a GPU: every kernel of the design against plain formulas, then the engine (fp32 and bf16) against the oracle over prompts,
portions, mixed batches, decoding, reused pages and slots, drafts, the scheduler and the trace program."""
import json
import math
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from mixed_stack_models import BLEND, CONFIGS, PLAIN, attention, dense, hgrn2, latent, make_tensors, model, write_snapshot
from stack_helpers import DEPTH, DEV, STEPS, Paged, i32, meta, rel, status_word

from cuteafd_b200 import ops
from cuteafd_b200.ref import mixed_stack as oracle
from cuteafd_b200.ref.hybrid_stack import rms_norm
from cuteafd_b200.ref.hyper_stack import attend, linear_attention, silu, visible

pytestmark = pytest.mark.gpu


def up(n, m=64):
    return -(-n // m) * m


# ------------------------------------------------------------------ kernels
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("W", [40, 1283, 9000])
def test_residual_rows(W, f32):
    """Scaled embedding rows, plain sums handed on as they are, normalised sums, the embedding added again, rows of unit norm."""
    torch.manual_seed(0)
    T, V, Wp, eps = 21, 50, up(W, 8), 0.3
    dt, tol = (torch.float32, 3e-6) if f32 else (torch.bfloat16, 4e-3)
    pad = lambda t: torch.nn.functional.pad(t, (0, Wp - W)).to(DEV).contiguous()
    table, toks, post = torch.randn(V, W).to(torch.bfloat16), torch.randint(0, V, (T,)), torch.randn(W)
    a, b = torch.randn(T, W).to(dt), torch.randn(T, W).to(dt)
    x, xn, st = torch.full((T, Wp), 3.0, device=DEV), torch.full((T, Wp + 8), 5.0, dtype=dt, device=DEV), status_word()
    kw, emb = dict(f32=f32, eps=eps, status=st), dict(tokens=i32(toks.tolist()), table=pad(table), scale=0.75)
    ops.norm_rows(x, W, T, xn=xn, **emb, **kw)
    want = table.float()[toks] * 0.75
    assert rel(x[:, :W], want) < 1e-6 and rel(xn[:, :W], oracle.unit_norm(want, eps)) < tol and float((xn[:, Wp:] - 5).abs().sum()) == 0
    ops.norm_rows(x, W, T, add=pad(a), xn=xn, raw=True, **kw)
    want = want + a.float()
    assert rel(x[:, :W], want) < 1e-6 and rel(xn[:, :W], want) < tol and float(x[:, W:].abs().sum()) == 0
    ops.norm_rows(x, W, T, add=pad(b), post=pad(post), xn=xn, **emb, **kw)
    want = want + rms_norm(b.float(), post, eps) + table.float()[toks] * 0.75
    assert rel(x[:, :W], want) < 2e-6 and rel(xn[:, :W], oracle.unit_norm(want, eps)) < tol
    rows, out = [5, 0, T - 1, 5], torch.zeros(4, Wp, dtype=dt, device=DEV)
    ops.norm_rows(x, W, 4, src_rows=i32(rows), xn=out, **kw)
    assert rel(out[:, :W], oracle.unit_norm(want[rows], eps)) < tol and int(st[0]) == 0
    ops.norm_rows(x, W, 1, add=pad(a), tokens=i32([V]), table=pad(table), **kw)           # a token outside the table is reported, not read
    assert int(st[0]) >> 24 == 5


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_side_gate(dt):
    torch.manual_seed(1)
    T, n, V = 37, 19, 30
    z, table, toks, st = torch.randn(T, 24) * 2, torch.randn(V, 5 * n).to(torch.bfloat16), torch.randint(0, V, (T,)), status_word()
    out = torch.full((T, 32), 5.0, dtype=dt, device=DEV)
    ops.side_gate(z.to(DEV), i32(toks.tolist()), table.to(DEV), 3 * n, n, out, T, status=st)
    want = oracle.gelu_tanh(z[:, :n]) * table.float()[toks][:, 3 * n:4 * n]
    assert rel(out[:, :n], want) < (1e-6 if dt == torch.float32 else 4e-3) and float((out[:, n:] - 5).abs().sum()) == 0 and int(st[0]) == 0


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("T", [3, 30, 300])
def test_products_with_an_output_factor(kind, T):
    """The factor multiplies every form of a product: plain, split over K, fp32 output, gated halves."""
    torch.manual_seed(2)
    N, K, dt = 200, 1024, torch.float32 if kind == "f32" else torch.bfloat16
    x, w, u = torch.randn(T, K).to(dt), (torch.randn(N, K) * K ** -0.5).to(dt), (torch.randn(N, K) * K ** -0.5).to(dt)
    W, U = (ops.TcWeight.from_master(m.float(), kind, DEV) for m in (w, u))
    W.alpha, U.alpha = torch.full((1,), 1.7, device=DEV), torch.full((1,), 0.6, device=DEV)
    tn = ops.pick_tn(T, swiglu=True)
    act = ops.ActBuffer.alloc(ops.KIND_BY_NAME[kind], T, K, tn, DEV)
    act.data.copy_(x)
    want, tol = 1.7 * x.float() @ w.float().T, 1e-5 if kind == "f32" else 4e-3
    for splits, out in ((1, dt), (1, torch.float32)) + (((4, dt), (2, torch.float32)) if kind == "bf16" else ()):
        y = torch.zeros(T, N, dtype=out, device=DEV)
        ops.tc_linear(W, act, y, rows=T, splits=splits)
        assert rel(y, want) < tol
    if kind == "bf16":
        y = torch.zeros(T, N, dtype=dt, device=DEV)
        ops.tc_linear(W, act, y, rows=T, w_up=U)
        assert rel(y, silu(want) * (0.6 * x.float() @ u.float().T)) < tol


def pooled_slot(pages, b, P):
    """(page, row in it) of block b: strips of eight blocks stand with the page of their first token, several of one page in order."""
    first = (b // 8) * 8 * P // 64
    strips = [s for s in range(b // 8 + 1) if s * 8 * P // 64 == first]
    return pages[first], strips.index(b // 8) * 8 + b % 8


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dim,vdim,rot,P,norm", [(6, 2, 40, 24, 12, 6, True), (3, 3, 33, 45, 22, 1, True), (4, 1, 128, 128, 128, 16, True), (4, 2, 192, 64, 32, 3, False), (2, 1, 256, 200, 64, 70, True),
                                                     (5, 5, 14, 72, 0, 8, True)])
def test_bias_rotation_unit_norm_and_pooled_blocks_across_portions(H, G, dim, vdim, rot, P, norm, f32):
    """Queries, cached rows and the means of every complete block, wherever the sequences are cut, after steps back and on pages that others used."""
    torch.manual_seed(3)
    dt, tol, eps, base = (torch.float32, 4e-6, 1e-3, 300.0) if f32 else (torch.bfloat16, 6e-3, 1e-3, 300.0)
    dp, dvp, C, L, slots = up(dim), up(vdim), (H + G) * dim + G * vdim, 240, [2, 0, 3]
    u, bias = [torch.randn(L, C).to(dt).float() for _ in slots], torch.randn(C)
    R, W = ops.pooled_page_rows(P), G * (dp + dvp)
    want = []
    for x in u:
        y = x + bias
        q, k, v = y[:, :H * dim].view(L, H, dim), y[:, H * dim:(H + G) * dim].view(L, G, dim), y[:, (H + G) * dim:].view(L, G, vdim)
        q, k = (oracle.turn(z, {"dims": rot, "base": base}, False) for z in (q, k))
        want.append((oracle.unit_norm(q, eps), oracle.unit_norm(k, eps), v) if norm else (q, k, v))
    n_pages = 14
    ids = (torch.randperm(n_pages - 1, generator=torch.Generator().manual_seed(4)) + 1).tolist()
    pages = [[ids.pop() for _ in range(4)] for _ in slots]
    table = i32(pages)
    cache, pooled = torch.full((n_pages * 64, W + 64), 9.0, dtype=dt, device=DEV), torch.full((n_pages * R, W), 9.0, dtype=dt, device=DEV)
    st, bd, done = status_word(), bias.to(DEV), [0, 0, 0]
    for runs in STEPS:
        T, longest = sum(n for _, n in runs), max(n for _, n in runs)
        pos = [p + i for p, n in runs for i in range(n)]
        where = [pages[s][(p + i) // 64] * 64 + (p + i) % 64 for s, (p, n) in enumerate(runs) for i in range(n)]
        proj = torch.full((T, up(C, 8) + 16), 77.0, dtype=dt, device=DEV)
        proj[:, :C] = torch.cat([u[s][p:p + n] for s, (p, n) in enumerate(runs)]).to(dt)
        ang = torch.tensor(pos, dtype=torch.float64)[:, None] * torch.tensor([base ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64)
        turn = torch.stack([ang.cos(), ang.sin()], -1).float().to(DEV) if rot else None
        q, m = torch.zeros(T, H * dp, dtype=dt, device=DEV), meta(runs, slots, where)
        m["page_table"] = table
        for rep in range(2 if longest <= DEPTH else 1):
            ops.conv_qkv(proj, None, None, None, turn, None, q, cache, m, H=H, G=G, dim=dim, dp=dp, vdim=vdim, dvp=dvp, pairs=rot // 2, eps=eps, n_seq=3, max_q_len=longest, bias=bd,
                         norm="head" if norm else "", half=True, n_slots=4, pooled=pooled, pool=P, status=st)
            ops.pool_kv(cache, pooled, P, table, m["kv_len"], m["q_len"], width=W, n_seq=3, max_q_len=longest, status=st)
        assert int(st[0]) == 0
        row = 0
        for s, (p, n) in enumerate(runs):
            got = q[row:row + n].view(n, H, dp)
            assert rel(got[..., :dim], want[s][0][p:p + n]) < tol and float(got[..., dim:].abs().sum()) == 0, runs
            c = cache[torch.tensor(where[row:row + n], device=DEV)]
            assert rel(c[:, :G * dp].view(n, G, dp)[..., :dim], want[s][1][p:p + n]) < tol and rel(c[:, G * dp:W].view(n, G, dvp)[..., :vdim], want[s][2][p:p + n]) < tol, runs
            row, done[s] = row + n, p + n
            blocks = done[s] // P
            if not blocks:
                continue
            at = [pg * R + r for pg, r in (pooled_slot(pages[s], b, P) for b in range(blocks))]
            held = torch.tensor([pages[s][i // 64] * 64 + i % 64 for i in range(blocks * P)], device=DEV)
            means = cache[held][:, :W].float().view(blocks, P, W).mean(1).cpu()
            z = pooled[torch.tensor(at, device=DEV)].float().cpu()
            for lo, w, d in ((0, dp, dim), (G * dp, dvp, vdim)):
                a, b = (x[:, lo:lo + G * w].view(blocks, G, w)[..., :d] for x in (z, means))
                assert rel(a, b) < (1e-6 if f32 else 4e-3) and float((a - b).abs().max()) < (1e-5 if f32 else 0.04), (runs, s)


@pytest.mark.parametrize("H,G,dim,vdim,window,P,splits", [
    (8, 1, 128, 72, 90, 8, 2), (3, 3, 40, 24, 1, 1, 3), (6, 2, 64, 64, 64, 16, 3), (9, 1, 200, 256, 65, 3, 4), (5, 1, 192, 33, 63, 20, 1), (40, 1, 100, 192, 130, 4, 5), (12, 4, 256, 128, 33, 2, 7),
    (128, 1, 16, 48, 100, 12, 6), (4, 2, 130, 136, 4096, 8, 7), (6, 3, 96, 96, 50, 70, 3), (2, 1, 64, 64, 7, 5, 2)])
def test_attention_over_pooled_blocks_and_a_window(H, G, dim, vdim, window, P, splits):
    """Ragged batch on scattered pages; rows point at the first key of their window, at the one just in front of it, at the last block that is seen and
    the next one, at blocks far back - the tcgen05 kernels and the ordinary-core one.  Slots nobody owns, and blocks not yet seen, hold large noise."""
    torch.manual_seed(5)
    lens, q_lens = [733, 64, 393, 1, 65], [130, 1, 2, 1, 65]
    dt, scale = torch.bfloat16, 0.7
    pg = Paged(lens, G, dim, vdim, dt)
    T, group, R, W = sum(q_lens), H // G, ops.pooled_page_rows(P), G * (pg.dp + pg.dvp)
    pooled = torch.randn(pg.store.shape[0] // 64 * R, W, generator=torch.Generator().manual_seed(6)) * 40
    for s, n in enumerate(lens):
        # tokens of a block share a direction, so that their mean stands out like a key of its own
        for b in range(n // P):
            pg.k[s][b * P:(b + 1) * P] = (pg.k[s][b * P] + 0.3 * pg.k[s][b * P:(b + 1) * P]).to(dt).float()
        pages = pg.table[s].tolist()
        at = torch.tensor([pages[j // 64] * 64 + j % 64 for j in range(n)], device=DEV)
        rows = torch.zeros(n, G, pg.dp)
        rows[..., :dim] = pg.k[s]
        pg.store[at, :G * pg.dp] = rows.view(n, -1).to(dt).to(DEV)
        for b in range(n // P):
            page, r = pooled_slot(pages, b, P)
            line = torch.zeros(W)
            line[:G * pg.dp].view(G, pg.dp)[:, :dim] = pg.k[s][b * P:(b + 1) * P].mean(0)
            line[G * pg.dp:].view(G, pg.dvp)[:, :vdim] = pg.v[s][b * P:(b + 1) * P].mean(0)
            if (b + 1) * P - 1 <= n - 1 - window:                        # the others are never seen: they stay noise
                pooled[page * R + r] = line
    starts = [sum(q_lens[:i]) for i in range(len(q_lens))]
    q = torch.zeros(T, H, pg.dp)
    q[..., :dim] = torch.randn(T, H, dim) * 0.1
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        for i in range(m):
            pos = n - m + i
            seen = max(0, pos - window + 1) // P
            keys = [pg.k[s][k] for k in (pos - window + 1, pos - window, pos - window + 2, pos - window - 1, 0, 63, 64, pos, pos - 1) if 0 <= k <= pos]
            keys += [pg.k[s][b * P:(b + 1) * P].mean(0) for b in (seen - 1, seen, 0, 7, 8, 63, 64) if 0 <= b and (b + 1) * P <= n]
            for h in range(H):
                if (i + h) % 5:
                    k = keys[(i * 3 + h) % len(keys)][h // group]
                    q[starts[s] + i, h, :dim] += k * (14.0 / float(k @ k))
    q = q.to(dt)
    qd, ldo, st, pooled = q.reshape(T, -1).to(DEV), up(H * vdim, 8), status_word(), pooled.to(dt).to(DEV)
    maps, pmaps = ops.encode_window_maps(pg.store, G, pg.dp, pg.dvp), ops.encode_window_maps(pooled, G, pg.dp, pg.dvp, box_rows=8)
    extras = ops.attn_extras(pooled=pooled, pool_maps=pmaps, pool=P)
    kw = dict(T=T, n_seq=len(lens), Hq=H, Hkv=G, dp=pg.dp, dvp=pg.dvp, dv=vdim, window=window, scale=scale, extras=extras, status=st)
    where = (pg.table, i32(lens), i32(starts), i32(q_lens))
    new = lambda: torch.full((T, ldo), 7.0, dtype=dt, device=DEV)
    outs = {"simt": new()}
    ops.window_attention_simt(qd, pg.store, *where, outs["simt"], pool_stride=W, **kw)
    for name, n in (("one", 1), ("split", splits)):
        po = torch.full((n * T * H * pg.dvp,), float("nan"), device=DEV)
        pml = torch.full((n * T * H * 2,), float("nan"), device=DEV)
        outs[name] = new()
        ops.window_attention(qd, maps, *where, outs[name], max_q_len=max(q_lens), n_splits=n, part_o=po, part_ml=pml, **kw)
    if pg.dp + 2 * pg.dvp <= 512:
        outs["prefill"] = new()
        ops.window_attention(qd, maps, *where, outs["prefill"], max_q_len=max(q_lens), prefill=True, **kw)
    assert int(st[0]) == 0
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        full = torch.zeros(n, H, dim)
        full[n - m:] = q[starts[s]:starts[s] + m, :, :dim].float()
        want = masked_pooled_attention(full, pg.k[s], pg.v[s], scale, window, P)[n - m:]
        for name, o in outs.items():
            o = o[starts[s]:starts[s] + m].float().cpu()
            err = (o[:, :H * vdim].reshape(m, H, vdim) - want).norm(dim=-1) / want.norm(dim=-1)
            assert float(err.max()) < 3e-2, (name, s, float(err.max()))
            assert float((o[:, H * vdim:] - 7).abs().sum()) == 0


def masked_pooled_attention(q, k, v, scale, window, P):
    """`oracle.pooled_attention` in one piece: tokens and means side by side under a mask."""
    n, T = k.shape[0] // P, q.shape[0]
    mean = lambda x: x[:n * P].reshape(n, P, *x.shape[1:]).mean(1)
    i = torch.arange(T)[:, None]
    see = torch.cat([visible(T, window, 0), (torch.arange(n)[None] + 1) * P - 1 <= i - window], 1)
    k, v, g = torch.cat([k, mean(k)]), torch.cat([v, mean(v)]), q.shape[1] // k.shape[1]
    s = torch.einsum("thd,jhd->htj", q, k.repeat_interleave(g, 1)) * scale
    return torch.einsum("htj,jhd->thd", torch.softmax(s.masked_fill(~see, -math.inf), -1), v.repeat_interleave(g, 1))


def test_masked_form_is_the_plain_one():
    torch.manual_seed(7)
    q, k, v = torch.randn(40, 4, 8), torch.randn(40, 2, 8), torch.randn(40, 2, 5)
    for window, P in ((1, 1), (7, 4), (40, 3), (5, 16)):
        assert torch.allclose(masked_pooled_attention(q, k, v, 0.5, window, P), oracle.pooled_attention(q, k, v, 0.5, window, P), atol=1e-5)


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,d,rot,r,rq", [(5, 40, 16, 72, 88), (3, 13, 6, 21, 19), (12, 128, 64, 512, 200), (2, 24, 72, 600, 33), (1, 33, 2, 65, 9)])
def test_latent_down_projections_and_query_heads(H, d, rot, r, rq, f32):
    torch.manual_seed(8)
    T, ldt, eps, base, n_slots = 21, 32, 1e-2, 50.0, 200
    dt, tol = (torch.float32, 3e-6) if f32 else (torch.bfloat16, 5e-3)
    rp, rotp, dp, q_col, kv_col = up(r), up(rot), up(d), 8, up(8 + rq, 8)
    proj, gq, gk = torch.randn(T, kv_col + r + rot + 5), torch.randn(rq), torch.randn(r)
    proj = torch.nn.functional.pad(proj, (0, -proj.shape[1] % 4))
    pos = torch.randint(0, 3000, (T,), generator=torch.Generator().manual_seed(1))
    ang = pos.double()[:, None] * torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
    cs = torch.stack([ang.cos(), ang.sin()], -1).float()
    where, st = torch.randperm(n_slots)[:T], status_word()
    cache, cq = torch.full((n_slots, rp + rotp + 64), 9.0, dtype=dt, device=DEV), torch.zeros(T, up(rq, 8), dtype=dt, device=DEV)
    pairs = lambda x: torch.stack([x[..., ::2] * cs[..., 0] - x[..., 1::2] * cs[..., 1], x[..., 1::2] * cs[..., 0] + x[..., ::2] * cs[..., 1]], -1).flatten(-2)
    ops.latent_down(proj.to(DEV), q_col, kv_col, gq.to(DEV), gk.to(DEV), cs.to(DEV), i32(where.tolist()), cq, cache, T=T, r=r, rp=rp, rot=rot, eps=eps, status=st)
    c = cache[where.to(DEV)].float().cpu()
    assert rel(cq[:, :rq], rms_norm(proj[:, q_col:q_col + rq], gq, eps)) < tol and rel(c[:, :r], rms_norm(proj[:, kv_col:kv_col + r], gk, eps)) < tol
    assert rel(c[:, rp:rp + rot], pairs(proj[:, kv_col + r:kv_col + r + rot])) < tol
    assert float(c[:, r:rp].abs().sum() + c[:, rp + rot:rp + rotp].abs().sum()) == 0 and float((c[:, rp + rotp:] - 9).abs().sum()) == 0
    q = torch.randn(T, up(H * (d + rot), 8)).to(dt)
    qn, qr = torch.zeros(H * ldt, dp, dtype=dt, device=DEV), torch.zeros(H * ldt, rotp, dtype=dt, device=DEV)
    tiles, n_tiles = torch.zeros(H * 2, 4, dtype=torch.int32, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.latent_split(q.to(DEV), cs.to(DEV), qn, qr, tiles, n_tiles, T=T, ldt=ldt, H=H, d=d, rot=rot, tn=16)
    heads = q[:, :H * (d + rot)].float().view(T, H, d + rot).transpose(0, 1)
    a, b = qn.view(H, ldt, dp).float().cpu(), qr.view(H, ldt, rotp).float().cpu()
    assert torch.equal(a[:, :T, :d], heads[..., :d]) and rel(b[:, :T, :rot], pairs(heads[..., d:])) < tol and float(a[..., d:].abs().sum() + b[..., rot:].abs().sum() + a[:, T:].abs().sum()) == 0
    assert int(n_tiles) == 2 * H and tiles.tolist() == [[h, h * ldt + 16 * j, 16 if j == 0 else 5, 0] for h in range(H) for j in range(2)] and int(st[0]) == 0


class LatentRows:
    """Paged latent rows with a rotated part: [latent, pad to 64 | rotated, pad to 64 | noise]."""

    def __init__(self, lens, r, rot, dt, seed=0):
        g = torch.Generator().manual_seed(seed)
        need = [-(-n // 64) for n in lens]
        ids = (torch.randperm(sum(need) + 2, generator=g) + 1).tolist()
        store = torch.randn((sum(need) + 3) * 64, up(r) + up(rot) + 64, generator=g) * 40
        self.c, self.k, table = [], [], torch.zeros(len(lens), max(need), dtype=torch.int32)
        for i, n in enumerate(lens):
            pages = [ids.pop() for _ in range(need[i])]
            table[i, :len(pages)] = torch.tensor(pages)
            c, k = torch.randn(n, r, generator=g).to(dt).float(), torch.randn(n, rot, generator=g).to(dt).float()
            at = torch.tensor([pages[j // 64] * 64 + j % 64 for j in range(n)])
            store[at, :up(r) + up(rot)] = 0
            store[at, :r] = c
            store[at, up(r):up(r) + rot] = k
            self.c.append(c); self.k.append(k)
        self.store, self.table = store.to(dt).to(DEV), table.to(DEV)


def pointed(rows, lens, q_lens, starts, H, ldt, r, rot, part):
    """Query rows (unrotated-space part, rotated part) most of which point at one key by its latent or - every other one - by its rotated part alone."""
    T = sum(q_lens)
    ql, qr = torch.zeros(H, ldt, r), torch.zeros(H, ldt, rot)
    ql[:, :T], qr[:, :T] = torch.randn(H, T, r) * 0.1, torch.randn(H, T, rot) * 0.1
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        for i in range(m):
            pos = n - m + i
            keys = [b for b in (0, 1, 62, 63, 64, 65, 127, 128, 129, 191, 192) if b <= pos] + [pos]
            for h in range(H):
                key = keys[(i * 7 + h) % len(keys)]
                if (i + h) % 4 == 1:
                    ql[h, starts[s] + i] += part(s, h, key)
                elif (i + h) % 4:
                    k = rows.k[s][key]
                    qr[h, starts[s] + i] += k * (16.0 / float(k @ k))
    return ql, qr


@pytest.mark.parametrize("H,r,rot,splits", [(3, 50, 64, 1), (4, 96, 32, 4), (6, 192, 16, 3), (16, 256, 64, 2), (1, 300, 8, 5), (24, 384, 64, 2), (5, 448, 2, 1), (128, 512, 64, 2), (40, 512, 48, 1)])
def test_absorbed_attention_with_a_rotated_part_and_sinks(H, r, rot, splits):
    torch.manual_seed(9)
    lens, q_lens, dt, scale = [333, 64, 193, 1, 65], [70, 1, 2, 1, 65], torch.bfloat16, 0.9
    T, ldt, rp = sum(q_lens), sum(q_lens) + 5, up(r)
    starts, pg = [sum(q_lens[:i]) for i in range(len(q_lens))], LatentRows(lens, r, rot, dt)
    ql, qr = pointed(pg, lens, q_lens, starts, H, ldt, r, rot, lambda s, h, key: pg.c[s][key] * (14.0 / float(pg.c[s][key] @ pg.c[s][key])))
    qlp, qrp = torch.zeros(H, ldt, rp), torch.zeros(H, ldt, 64)
    qlp[..., :r], qrp[..., :rot] = ql, qr
    qlp, qrp, sink = qlp.to(dt), qrp.to(dt), torch.randn(H) * 2 + 3.0
    from cuteafd_b200.ops.native import call
    host = torch.zeros(128, dtype=torch.uint8)
    call("cuteafd_tmap_encode_latent_rows", host.data_ptr(), pg.store.data_ptr(), pg.store.shape[0], rp + 64, pg.store.shape[1])
    st, sd = status_word(), sink.to(DEV)
    po, pml = torch.full((splits * T * H * rp,), float("nan"), device=DEV), torch.full((splits * T * H * 2,), float("nan"), device=DEV)
    new = lambda: torch.full((H * ldt, rp), 7.0, dtype=dt, device=DEV)
    tc, simt, qd, rd = new(), new(), qlp.reshape(H * ldt, rp).to(DEV), qrp.reshape(H * ldt, 64).to(DEV)
    where, kw = (pg.table, i32(lens), i32(starts), i32(q_lens), None), dict(T=T, ldt=ldt, n_seq=len(lens), H=H, rank_pad=rp, scale=scale, q_rope=rd, sink=sd, status=st)
    ops.latent_attention(qd, host.to(DEV), *where, tc, max_q_len=max(q_lens), n_splits=splits, part_o=po, part_ml=pml, **kw)
    ops.latent_attention_simt(qd, pg.store, *where, simt, **kw)
    assert int(st[0]) == 0
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        rows = slice(starts[s], starts[s] + m)
        full = torch.zeros(n, H, r + rot)
        full[n - m:] = torch.cat([qlp[:, rows, :r], qrp[:, rows, :rot]], -1).float().transpose(0, 1)
        keys = torch.cat([pg.c[s], pg.k[s]], 1)[:, None]
        want = attend(full, keys, pg.c[s][:, None], scale, visible(n, None, 0), sink)[n - m:]
        ref = want.norm(dim=-1) + 0.2 * attend(full, keys, pg.c[s][:, None], scale, visible(n, None, 0), None)[n - m:].norm(dim=-1)
        for o in (tc, simt):
            o = o.view(H, ldt, rp)[:, rows].float().cpu().transpose(0, 1)
            assert float(((o[..., :r] - want).norm(dim=-1) / ref).max()) < 2e-2, s
            assert rp == r or float(o[..., r:].abs().max()) == 0
    assert float((tc.view(H, ldt, rp)[:, T:].float() - 7).abs().max()) == 0


@pytest.mark.parametrize("H,d,rot,dv,r", [(3, 40, 16, 24, 72), (2, 128, 64, 128, 512), (5, 64, 2, 65, 100), (4, 192, 64, 80, 256), (2, 100, 48, 100, 64), (1, 1, 2, 1, 8)])
def test_expanding_prefill_attention_with_a_rotated_part_and_sinks(H, d, rot, dv, r):
    from cuteafd_b200.ops.native import call, ptr, stream
    torch.manual_seed(10)
    lens, q_lens, dt, scale = [400, 131, 64], [200, 131, 1], torch.bfloat16, 0.8
    rp, dp, dvp, row = up(r), up(d), up(dv), up(r) + 64
    pg = LatentRows(lens, r, rot, dt)
    T, ldt, starts, ctx, tot = sum(q_lens), sum(q_lens) + 3, [0, 200, 331], [], 0
    for n in lens:
        ctx.append(tot)
        tot += up(n)
    uk, uv = (torch.randn(H, d, r) * r ** -0.5).to(dt).float(), (torch.randn(H, dv, r) * r ** -0.5).to(dt).float()

    def by_latent(s, h, key):
        k = uk[h] @ pg.c[s][key]
        return k * min(12.0 / float(k @ k), 20.0)
    qn, qr = pointed(pg, lens, q_lens, starts, H, ldt, d, rot, by_latent)
    q, q2 = torch.zeros(H, ldt, dp), torch.zeros(H, ldt, 64)
    q[..., :d], q2[..., :rot] = qn, qr
    q, q2, sink, st = q.to(dt), q2.to(dt), torch.randn(H) * 2 + 2.0, status_word()
    kvw = torch.zeros(H, dp + dvp, rp)
    kvw[:, :d, :r], kvw[:, dp:dp + dv, :r] = uk, uv
    w = ops.TcWeight.from_master(kvw.reshape(H * (dp + dvp), rp), "bf16", DEV)
    cap = tot + 64
    lat, kvb = torch.zeros(cap, row, dtype=dt, device=DEV), torch.zeros(cap, H * (dp + dvp), dtype=dt, device=DEV)
    out = torch.full((T, up(H * dv, 8)), 7.0, dtype=dt, device=DEV)
    kl, qs, ql, cx, sd = i32(lens), i32(starts), i32(q_lens), i32(ctx), sink.to(DEV)
    call("cuteafd_latent_gather_ctx", ptr(pg.store), ptr(pg.table), ptr(cx), ptr(kl), ptr(lat), 3, max(lens), pg.table.shape[1], pg.store.shape[0], cap, row, pg.store.shape[1], ptr(st), stream())
    view = lat[:, :rp]
    ops.tc_linear(w, ops.ActBuffer(ops.KIND_BF16, cap, rp, 256, view, ops.encode_tmap(view, 256)), kvb, rows=tot, status=st)
    qd, rd = q.reshape(H * ldt, dp).to(DEV), q2.reshape(H * ldt, 64).to(DEV)
    call("cuteafd_latent_prefill_attention", ptr(qd), ptr(rd), ptr(kvb), ptr(lat), row, rp, ptr(sd), cap, ptr(cx), ptr(kl), ptr(qs), ptr(ql), None, ptr(out), T, ldt, 3, max(q_lens), H, dp, dvp, dv,
         out.shape[1], scale, ptr(st), stream())
    assert int(st[0]) == 0
    got = out.float().cpu()
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        for h in range(H):
            k, v, rows = torch.cat([pg.c[s] @ uk[h].T, pg.k[s]], 1), pg.c[s] @ uv[h].T, slice(starts[s], starts[s] + m)
            sc = torch.cat([q[h, rows, :d], q2[h, rows, :rot]], -1).float() @ k.T * scale
            see = torch.arange(n)[None] <= (n - m + torch.arange(m))[:, None]
            want = oracle.sink_softmax(sc.masked_fill(~see, -math.inf), sink[h]) @ v
            o = got[rows, h * dv:(h + 1) * dv]
            assert rel(o, want) < 2e-2 and float((o - want).abs().max()) < 0.06 * float(want.abs().max()), (s, h)
    assert float((got[:, H * dv:] - 7).abs().sum()) == 0


def scan_buffers(H, d, dv, n_state=4):
    vp = -(-dv // 4) * 4
    g = torch.Generator(device=DEV).manual_seed(3)
    state = torch.empty(n_state, 2, H, d, vp, device=DEV).normal_(0, 30, generator=g)
    tags = torch.randint(-1, 300, (n_state, H, 2), dtype=torch.int32, device=DEV, generator=g)
    return state, tags, torch.empty(n_state, DEPTH, H, 2 * d + vp, device=DEV).normal_(0, 30, generator=g)


SHORT, CHUNKS, FP32 = "short", "chunks", "fp32"
LONG_STEPS = [[(0, 400), (0, 2), (0, 17)], [(400, 3), (2, 300), (17, 128)], [(403, 256), (302, 1), (145, 129)], [(659, 1), (303, 270), (274, 8)], [(660, 33), (573, 130), (276, 385)]]


@pytest.mark.parametrize("form", [FP32, SHORT, CHUNKS])
@pytest.mark.parametrize("H,d,dv,gates", [(3, 24, 40, "mild"), (1, 13, 7, "long"), (2, 128, 256, "mild"), (4, 64, 64, "harsh"), (2, 128, 128, "long"), (3, 9, 17, "harsh"), (2, 256, 64, "mild"),
                                          (2, 96, 200, "harsh"), (2, 128, 64, "harsh"), (2, 128, 64, 0.0), (2, 64, 128, -2.0), (3, 40, 40, -3.0), (2, 128, 256, -5.0), (2, 100, 72, -7.0)])
def test_hgrn2_across_portions(H, d, dv, gates, form):
    """Gates, recurrence and output norm of every portion equal those of the whole sequence, wherever it is cut and after steps back.  "long": every
    channel remembers for thousands of tokens; "harsh": channels that forget at once, beside ones that forget nothing, without lower bounds; a number:
    gates around it without lower bounds, which take more and more references in a chunk."""
    torch.manual_seed(11)
    f32 = form == FP32
    dt, tol, eps = torch.float32 if f32 else torch.bfloat16, 1e-5 if f32 else 8e-3, 1e-3
    slots, L = [1, 3, 0], 704
    bias, lower = (torch.randn(H * d) * 0.3 + gates, torch.zeros(H * d)) if isinstance(gates, float) else {"mild": (torch.randn(H * d) * 1.5 + 1.0, torch.rand(H * d) * 0.9), "long": (torch.randn(H * d) * 0.5 + 9.0, torch.zeros(H * d)),
                   "harsh": (torch.randn(H * d) * 4, torch.zeros(H * d))}[gates]
    if gates == "harsh":
        bias[0], bias[H * d - 1], lower[1] = 40.0, -60.0, 1.0        # forgets nothing and takes nothing; forgets at once; bound at one
    norm = torch.randn(dv) + 1.0
    widths = {"q": H * d, "z": H * d, "v": H * dv}
    at, cols = 8, {}
    for n, w in widths.items():
        cols[n], at = at, at + up(w, 8)
    seqs, want = [], []
    for _ in slots:
        x = {n: torch.randn(L, w).to(dt).float() for n, w in widths.items()}
        f = oracle.forget_gate(x["z"].double() + bias.double(), lower.double())
        keep = (1.0 - lower.double()) * torch.sigmoid(-(x["z"].double() + bias.double()))
        o = linear_attention(silu(x["q"].double()).view(L, H, d), keep.view(L, H, d), x["v"].double().view(L, H, dv), f.view(L, H, d))
        seqs.append(x)
        want.append(rms_norm(o, norm.double(), eps).reshape(L, -1).float())
    bd, ld, nd = bias.to(DEV), lower.to(DEV), norm.to(DEV)
    state, tags, ring = scan_buffers(H, d, dv)
    st = status_word()
    scratch = ops.scan_scratch(600, 3, H, d, dv, DEV) if form == CHUNKS and d <= 128 else None
    if scratch:
        scratch[0].fill_(float("nan")); scratch[1].fill_(float("nan"))
    back = [[(194, 8), (79, 8), (221, 8)], [(195, 30), (86, 9), (222, 1)]]                   # long runs behind rejected rows
    for runs in STEPS + back + [[(0, 1), (0, 17), (0, 400)]] + LONG_STEPS:
        T = sum(n for _, n in runs)
        proj = torch.full((T, at), 77.0, dtype=dt, device=DEV)
        for n, w in widths.items():
            proj[:, cols[n]:cols[n] + w] = torch.cat([seqs[s][n][p:p + m] for s, (p, m) in enumerate(runs)]).to(dt)
        out = torch.full((T, up(H * dv, 8) + 8), 5.0, dtype=dt, device=DEV)
        for rep in range(2 if max(n for _, n in runs) <= DEPTH else 1):
            arg = ops.decay_scan_arg(*(proj[:, cols[n]:] for n in ("q", "z", "v")), None, state, tags, ring, out, meta(runs, slots), H=H, dim=d, vdim=dv, n_seq=3,
                                     max_q_len=max(n for _, n in runs), eps=eps, forget=(bd, ld), norm=nd, chunks=scratch, T=T, status=st)
            ops.decay_scan(arg, f32=f32)
        assert int(st[0]) == 0, runs
        row = 0
        for s, (p, n) in enumerate(runs):
            e = (out[row:row + n, :H * dv].float().cpu() - want[s][p:p + n]).view(n, H, dv).norm(dim=-1) / want[s].view(L, H, dv).norm(dim=-1).mean(0)
            assert float(e.max()) < 3 * tol, (runs, s, float(e.max()))
            row += n
        assert float((out[:, H * dv:] - 5).abs().sum()) == 0


# ------------------------------------------------------------------ engine
def logits(cfg, t, toks):
    return oracle.logits(cfg, {k: v.double() for k, v in t.items()}, toks).float()


def build(cfg, tmp_path, dtype="float32", seed=0, max_tokens=2048, live=4, tensors=None):
    from cuteafd_b200.serving.trace import TraceReplay
    t = tensors or make_tensors(cfg, seed)
    p = write_snapshot(cfg, t, tmp_path / f"{dtype}{seed}")
    rep = TraceReplay(str(p), dtype=dtype, max_tokens=max_tokens, max_live=live)
    g = torch.Generator(device=DEV).manual_seed(9)      # what earlier owners of a page or a state slot could have left behind: large, finite
    for buf in rep.engine.cache_buffers() + rep.engine.state_buffers():
        buf.normal_(0, 30, generator=g) if buf.is_floating_point() else buf.random_(0, 60, generator=g)
    return rep, t


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_portions(rep, rid, toks, cuts, end=True):
    """Feeds `toks` in portions of the given sizes (the last one repeats); returns logits of every position."""
    out, at, i = [], 0, 0
    while at < len(toks):
        part = toks[at:at + cuts[min(i, len(cuts) - 1)]]
        at, i = at + len(part), i + 1
        out.append(rep.step([{"id": rid, "tokens": part, "want": list(range(len(part)))}], [rid] if end and at == len(toks) else []))
    rep.engine.check_status()
    return torch.cat(out)


def errors(got, want):
    """Per position: rms difference of the centred logits over their scale."""
    d = got - want
    return (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std()


def check(got, want, dtype):
    e = errors(got, want)
    if dtype == "float32":
        assert float(e.max()) < 1e-4, float(e.max())
    else:      # (norms over a few values divide by what may be nearly zero: there rounding turns whole rows)
        assert int((e > 0.2).sum()) <= max(1, len(e) // 100) and float(e.median()) < 0.04, (float(e.max()), float(e.median()), int((e > 0.2).sum()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompts_portions_and_decoding_match_the_oracle(name, dtype, tmp_path):
    cfg = CONFIGS[name]
    rep, t = build(cfg, tmp_path, dtype)
    toks = tokens(cfg, 230, 1)
    want = logits(cfg, t, toks)
    rep.engine.tap = [] if dtype == "float32" else None
    check(run_portions(rep, "a", toks, [len(toks)]), want, dtype)
    if dtype == "float32":
        taps, ref = rep.engine.tap, [x.float() for x in oracle.hidden_states(cfg, {k: v.double() for k, v in t.items()}, toks)]
        assert len(taps) == len(ref) and all(rel(a, b) < 1e-5 for a, b in zip(taps, ref))
        rep.engine.tap = None
    for i, cuts in enumerate(([160, 1], [2, 2, 3, 57, 64, 2, 63, 2, 9, 8, 7, 1, 65], [1], [64, 64, 1], [33], [130, 98, 2], [230])):
        check(run_portions(rep, f"p{i}", toks, cuts), want, dtype)
    assert rep.pool.n_free == rep.pool.n_pages - 1 and len(rep.runner._free_slots) == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_equal_each_alone_and_pages_and_slots_are_reused(dtype, tmp_path):
    cfg = BLEND
    rep, t = build(cfg, tmp_path, dtype, max_tokens=64 * 9)
    reqs = {"a": tokens(cfg, 150, 2), "b": tokens(cfg, 9, 3), "c": tokens(cfg, 70, 4), "d": tokens(cfg, 129, 5)}
    ref = {k: logits(cfg, t, v) for k, v in reqs.items()}
    plans = [{"a": 128, "b": 1}, {"b": 1, "c": 29}, {"a": 2, "b": 1, "c": 1}, {"b": 2, "c": 3}, {"a": 1, "b": 1, "d": 61}, {"d": 3, "a": 1}, {"a": 1, "b": 1, "c": 1, "d": 1},
             {"a": 1, "b": 1, "c": 1, "d": 1}]
    for rnd in range(3):                                     # freed pages and slots are taken again by the next pass, in another order
        got, at = {k: [] for k in reqs}, {k: 0 for k in reqs}
        steps = list(plans)
        while any(at[k] < len(v) for k, v in reqs.items()):
            plan = steps.pop(0) if steps else {k: 16 + 5 * rnd for k in reqs}
            entries, end = [], []
            for k, n in plan.items():
                part = reqs[k][at[k]:at[k] + n]
                if not part:
                    continue
                at[k] += len(part)
                entries.append((k, part))
                if at[k] == len(reqs[k]):
                    end.append(f"{k}{rnd}")
            order = entries if rnd % 2 == 0 else entries[::-1]
            out = rep.step([{"id": f"{k}{rnd}", "tokens": p, "want": list(range(len(p)))} for k, p in order], end)
            o = 0
            for k, p in order:
                got[k].append(out[o:o + len(p)])
                o += len(p)
        rep.engine.check_status()
        for k in reqs:
            check(torch.cat(got[k]), ref[k], dtype)
        assert rep.pool.n_free == rep.pool.n_pages - 1 and len(rep.runner._free_slots) == 4


WINDOW, POOL = 100, 12


def pointing(kind):
    """One layer whose second head, at rows of token 6, looks for token 5: two channels that only these tokens have decide its scores, in a dimension
    that does not turn.  Every other token's rows are the same to it."""
    layer = attention(2, 1, 40, 40, 2.0, 12, WINDOW, POOL) if kind == "attention" else latent(2, 24, 8, 24, 32, 32, 0.5)
    cfg = model(61, 96, [layer], side=0, scale=1.0)
    t = make_tensors(cfg, 7)
    p = "l0.mix"
    t["embed"][5] = torch.roll(t["embed"][7], 11)
    t["embed"][:, :2] = 0
    t["embed"][5, 0], t["embed"][6, 1] = 4.0, 4.0
    if kind == "attention":
        for k, row, ch in (("q", 40 + 39, 1), ("k", 39, 0)):
            t[f"{p}.{k}"][:, :2], t[f"{p}.{k}"][row], t[f"{p}.{k}.b"][row] = 0, 0, 0
            t[f"{p}.{k}"][row, ch] = 30.0
    else:
        for n, row, ch in (("dq", 31, 1), ("dkv", 31, 0)):           # the latents' last value carries the mark
            t[f"{p}.{n}"][:, :2], t[f"{p}.{n}"][row], t[f"{p}.{n}.norm"][31] = 0, 0, 2.0
            t[f"{p}.{n}"][row, ch] = 30.0
        for n, rows in (("uq", 32 + 23), ("uk", 24 + 23)):
            t[f"{p}.{n}"][:, 31], t[f"{p}.{n}"][rows] = 0, 0
            t[f"{p}.{n}"][rows, 31] = 2.0
        t[f"{p}.sink"][:] = 1.0
    return cfg, {k: v.to(torch.bfloat16).float() for k, v in t.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_one_key_decides_inside_the_window_or_its_block(kind, dtype, tmp_path):
    """One score stands out: a key just inside the window, or in a block that is just seen, must count; one just outside whose block is not yet seen must
    not - in prompts, portions and decoding, next to page borders too."""
    cfg, t = pointing(kind)
    rep, t = build(cfg, tmp_path, dtype, tensors=t)
    n = 300
    base = [x if x not in (5, 6) else 7 for x in tokens(cfg, n, 8)]
    seen = {True: 0, False: 0}
    for q in (WINDOW + POOL - 2, WINDOW + POOL - 1, 191, 192, 255, 256, 298):
        base_q = list(base)
        base_q[q] = 6
        alone = logits(cfg, t, base_q)
        edge = (q - WINDOW + 1) // POOL * POOL                # first token of the first block that is not seen
        for k in (q - WINDOW + 1, q - WINDOW, edge, edge - 1, edge - POOL, 0, q - 1):
            if not 0 <= k < q:
                continue
            toks = list(base_q)
            toks[k] = 5
            want = logits(cfg, t, toks)
            moved, inside = float(errors(alone[q:q + 1], want[q:q + 1])), kind == "latent" or q - k < WINDOW or k < edge
            assert moved > 0.1 if inside else moved < 1e-6, (q, k, moved)
            seen[inside] += 1
            for cuts in ([n], [q, 1, 2], [q - 1, 2]):
                got = run_portions(rep, "x", toks, cuts)
                e = float(errors(got[q:q + 1], want[q:q + 1]))
                assert e < (1e-4 if dtype == "float32" else 0.04), (q, k, cuts, e)
    assert seen[True] > 10 and (kind == "latent" or seen[False] > 5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sinks_take_their_share(dtype, tmp_path):
    """A head whose sink outweighs everything gives nothing, one without a share gives all."""
    cfg = model(61, 64, [latent(2, 16, 8, 16, 24, 24, 0.3)], side=0)
    t = make_tensors(cfg, 12)
    toks = tokens(cfg, 150, 13)
    outs = []
    for name, sink in (("all", [-60.0, -60.0]), ("one", [-60.0, 60.0]), ("half", [8.0, 8.0])):
        ts = dict(t, **{"l0.mix.sink": torch.tensor(sink)})
        rep, _ = build(cfg, tmp_path / name, dtype, tensors=ts)
        outs.append(logits(cfg, ts, toks))
        for cuts in ([150], [130, 1], [7]):
            check(run_portions(rep, "a", toks, cuts), outs[-1], dtype)
    assert all(float(errors(a, b).median()) > 0.05 for a, b in ((outs[0], outs[1]), (outs[0], outs[2]), (outs[1], outs[2])))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_token_is_remembered_for_hundreds_of_tokens(dtype, tmp_path):
    """A recurrence that forgets next to nothing, in a loop: the first token still shows at the end, through whole prompts, portions and decoding; a
    state that is lost, or taken from another pass or slot, would too."""
    cfg = model(61, 64, [hgrn2(2, 16, 16)], side=0, scale=1.0, loop=(0, 1, 2))
    t = make_tensors(cfg, 17)
    # a token takes a place in the state only in one channel, which token 5 opens (and nothing closes again); its value is far larger than the others'
    t["embed"][:, :2], t["embed"][:, 1] = 0, 2.0
    t["embed"][5, 0] = 6.0
    p = "l0.mix"
    t[f"{p}.lower"][:], t[f"{p}.f"][:], t[f"{p}.f.b"][:] = 0, 0, 9.0
    t[f"{p}.f"][:, 0] = -4.0
    t[f"{p}.q"] *= 0.2
    t[f"{p}.q"][:, 1] = 1.0
    t[f"{p}.v"][:, 0] = torch.randn(32, generator=torch.Generator().manual_seed(3)) * 6.0
    t = {k: v.to(torch.bfloat16).float() for k, v in t.items()}
    rep, t = build(cfg, tmp_path, dtype, tensors=t)
    toks = [x if x != 5 else 7 for x in tokens(cfg, 400, 18)]
    other = [5] + toks[1:]
    want, with5 = logits(cfg, t, toks), logits(cfg, t, other)
    assert float(errors(with5[380:], want[380:]).min()) > 0.08
    for cuts in ([400], [390, 1], [63, 2, 64, 65, 1, 128, 9, 8, 60], [100, 100]):
        a, b = run_portions(rep, "a", toks, cuts, end=False), run_portions(rep, "b", other, cuts, end=False)
        check(a, want, dtype)
        check(b, with5, dtype)
        rep.step([], ["a", "b"])


def test_first_tokens_and_single_token_prompts(tmp_path):
    for name in sorted(CONFIGS):
        rep, t = build(CONFIGS[name], tmp_path / name, "float32")
        for n in (1, 2, 3):
            toks = tokens(CONFIGS[name], n, 20 + n)
            check(run_portions(rep, f"r{n}", toks, [n]), logits(CONFIGS[name], t, toks), "float32")


@pytest.mark.parametrize("name", ["wide", "blend"])
def test_long_decoding_crosses_pages_windows_blocks_and_split_counts(name, tmp_path):
    cfg = CONFIGS[name]
    rep, t = build(cfg, tmp_path, "bfloat16")
    toks = tokens(cfg, 400, 30)
    check(run_portions(rep, "a", toks, [40, 1]), logits(cfg, t, toks), "bfloat16")
    assert rep.engine.graph_captures >= 1                     # decode steps replay captured graphs


def test_tokens_can_be_taken_back(tmp_path):
    """A step of up to `state_depth` rows may be continued from any of its rows: rejected rows leave no trace - in states or in blocks that they had
    completed - and a repeated step none either."""
    from cuteafd_b200.engine.kv import SeqKV
    from cuteafd_b200.serving.scheduler import Request, Row, SeqState
    cfg = BLEND
    rep, t = build(cfg, tmp_path)
    toks, wrong = tokens(cfg, 160, 31), tokens(cfg, 160, 32)
    want = logits(cfg, t, toks)
    st = SeqState(Request("a", list(toks)), SeqKV())
    run = lambda tk, pos: (rep.runner.run([Row(st, tk, pos, list(range(len(tk))))]), rep.runner.last_lane.logits[:len(tk)].cpu())[1]
    pos = 0
    for keep, drafted in ((2, 8), (66, 66), (3, 8), (1, 2), (7, 8), (8, 8), (1, 8), (1, 8), (1, 8), (2, 5), (4, 7), (1, 1), (5, 8), (1, 8), (1, 8), (1, 8)):
        rows = toks[pos:pos + keep] + wrong[pos + keep:pos + drafted]
        check(run(rows, pos)[:keep], want[pos:pos + keep], "float32")
        pos += keep
    check(run(toks[pos:], pos), want[pos:], "float32")
    with pytest.raises(RuntimeError, match="step back"):
        run(toks[pos:pos + 1], pos)
    rep.engine.check_status()


def test_greedy_generation_through_generate_and_the_scheduler(tmp_path):
    """The public generation call, and the scheduler with drafts, emit the oracle's greedy tokens (fp32 engine)."""
    import argparse

    from cuteafd_b200.cli import build_serving
    from cuteafd_b200.engine.generate import BatchGenerator, generate
    from cuteafd_b200.engine.registry import build_engine, load_weights, model_spec
    from cuteafd_b200.serving.scheduler import Request
    cfg = BLEND
    t = make_tensors(cfg, 11)
    p = str(write_snapshot(cfg, t, tmp_path / "m"))
    prompts = [tokens(cfg, n, 40 + n) for n in (67, 5, 100)]
    prompts.append([3, 1, 4, 1, 5] * 9)                       # repeats itself: the n-gram drafter has something to propose
    want = [oracle.greedy(cfg, t, q, 10)[0] for q in prompts]
    spec = model_spec(p, dtype="float32")
    eng = build_engine(spec, load_weights(p, spec, torch.device(DEV)), n_pages=16, max_seqs=4, max_pages_per_seq=8)
    assert generate(eng, prompts, 10) == want
    assert generate(eng, prompts[::-1], 10) == want[::-1]    # pages and state slots of the first call are used again
    g = BatchGenerator(eng, prefill_chunk=48)                # several chunks per prompt, none of them waiting for logits
    first = g.prefill(prompts)
    assert first == [w[0] for w in want] and g.decode_step() == [w[1] for w in want]
    ns = argparse.Namespace(model=p, device=0, dtype="float32", max_context=4096, max_sequences=3, pool_tokens=64 * 24, prefill_batch_tokens=50, decode_share=0.3,
                            prefix_cache_entries=8, prefix_cache_min_tokens=64, draft="ngram", draft_limit=12, layers=0, host_cache_gib=0.0)
    spec2, sched = build_serving(ns)
    assert spec2 == spec and sched.prefix is None and sched.max_draft == 7
    out = {}
    for i, q in enumerate(prompts):
        sched.submit(Request(f"r{i}", q, max_tokens=10, on_token=lambda tk, fin, why, i=i: out.setdefault(i, []).extend(tk)))
    sched.run_until_idle()
    assert [out[i] for i in range(4)] == want and sched.stats["drafted"] > 0


def test_random_weights_of_a_named_shape_run():
    """The synthetic preset at a small size: prefill and decode through the generator, bf16."""
    from cuteafd_b200.config import sikazen_spec
    from cuteafd_b200.engine.generate import generate
    from cuteafd_b200.engine.registry import build_engine
    from cuteafd_b200.models.mixed_stack import mixed_weights_random
    spec = sikazen_spec(n_layers=4, hidden=256, heads=4, kv_heads=2, ff=512, window=128, pool=8, rank=128, q_rank=96, rec_heads=2, rec_dim=64, rec_vdim=128, side=32, loop=(1, 3, 2))
    eng = build_engine(spec, mixed_weights_random(spec, torch.device(DEV)), n_pages=24, max_seqs=2, max_pages_per_seq=8)
    prompts = [torch.randint(0, spec.vocab, (n,), generator=torch.Generator().manual_seed(n)).tolist() for n in (200, 90)]
    a, b = generate(eng, prompts, 4), [generate(eng, [p], 4)[0] for p in prompts]
    assert all(len(x) == 4 for x in a) and sum(x == y for r, s in zip(a, b) for x, y in zip(r, s)) >= 6      # (a close pair of logits may turn)


def test_trace_program_end_to_end(tmp_path):
    cfg = PLAIN
    t = make_tensors(cfg, 13)
    p = write_snapshot(cfg, t, tmp_path / "m")
    a, b = tokens(cfg, 80, 60), tokens(cfg, 5, 61)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[70:72], "want": [0, 1]}, {"id": "b", "tokens": b, "want": [4, 0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[72:], "want": [7]}], "end": ["a", "b"]}]
    root = Path(__file__).resolve().parent.parent
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(p), "--dtype", "float32", "--out", str(out), "--max-tokens", "192"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300, env={**os.environ, "PATH": f"{Path(sys.executable).parent}:{os.environ['PATH']}"})
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = logits(cfg, t, a), logits(cfg, t, b)
    read = lambda n, rows: torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(rows, cfg["vocab"])
    check(torch.cat([read(1, 4), read(2, 1)]), torch.stack([wa[70], wa[71], wb[4], wb[0], wa[79]]), "float32")
    assert sorted(x.name for x in out.iterdir()) == ["1.f32", "2.f32"]

"""Latent-attention stacks on a GPU: every kernel of the design against plain fp32 formulas, then the engine (fp32 and bf16) against the
oracle over prompts, portions, mixed batches, decoding, reused pages, the scheduler and the trace program."""
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from latent_stack_models import CONFIGS, MIXED, ODD, ONCE, WIDE, make_tensors, masters_of, variant, write_snapshot

from cuteafd_b200 import ops
from cuteafd_b200.config import from_hf_config
from cuteafd_b200.ref import latent_stack as oracle

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def rel(got, want):
    return float((got.float().cpu() - want).norm() / want.norm())


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------ kernels
@pytest.mark.parametrize("f32", [True, False])
def test_row_kernels(f32):
    torch.manual_seed(0)
    T, W, V, P, k = 37, 1288, 50, 20, 11
    dt = torch.float32 if f32 else torch.bfloat16
    tol = 1e-6 if f32 else 4e-3
    table, pos = torch.randn(V, W).to(torch.bfloat16), torch.randn(P, W).to(torch.bfloat16)
    toks, positions = torch.randint(0, V, (T,)), torch.randint(0, P, (T,))
    w, b, alpha = torch.randn(W), torch.randn(W), 0.37
    wd, bd = w.to(DEV), b.to(DEV)
    x, cat, xn = torch.zeros(T, W, device=DEV), torch.zeros(T, 2 * W, dtype=dt, device=DEV), torch.zeros(T, W, dtype=dt, device=DEV)
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    ops.stack_embed(i32(toks.tolist()), i32(positions.tolist()), table.to(DEV), pos.to(DEV), x, cat[:, W:], ops.emit_arg(cat=cat), T, f32=f32, status=status)
    want = table.float()[toks] + pos.float()[positions]
    assert torch.equal(x.cpu(), want) and torch.equal(cat.cpu(), torch.cat([want, want], 1).to(dt)) and int(status[0]) == 0
    vec = torch.randn(W)
    ops.stack_stream(x, ops.emit_arg(norm=(wd, bd, alpha), xn=xn), T, f32=f32, vec=vec.to(DEV))
    want = want + vec
    assert torch.equal(x.cpu(), want) and rel(xn, oracle.dyt_norm(want, alpha, w, b)) < tol
    rows = [5, 0, 36, 5]
    out = torch.zeros(4, W, dtype=dt, device=DEV)
    ops.stack_stream(x, ops.emit_arg(norm=(wd, bd, alpha), xn=out), 4, f32=f32, src_rows=i32(rows))
    assert rel(out, oracle.dyt_norm(want[rows], alpha, w, b)) < tol
    mix, y = torch.randn(T, W).to(dt), torch.randn(T * k, W).to(dt)
    slot, wts = torch.randperm(T * k).reshape(T, k).int(), torch.rand(T, k)
    slot[3, 2] = -1                                          # a route that went nowhere
    ls1, ls2 = torch.randn(W), torch.randn(W)
    cat.zero_()
    ops.stack_combine(x, mix.to(DEV), ls1.to(DEV), y.to(DEV), slot.to(DEV), wts.to(DEV), ls2.to(DEV), ops.emit_arg(cat=cat), T, k)
    live = (slot >= 0).float()
    want = want + ls1 * mix.float() + ls2 * ((wts * live)[:, :, None] * y.float()[slot.clamp(min=0).long()]).sum(1)
    assert rel(x, want) < 1e-6 and rel(cat[:, :W], want) < tol and float(cat[:, W:].abs().max()) == 0
    ops.stack_combine(x, mix.to(DEV), ls1.to(DEV), None, None, None, None, None, T, 0)          # a layer without feed-forward
    assert rel(x, want + ls1 * mix.float()) < 1e-6


@pytest.mark.parametrize("f32,H,d,r,E,gate", [(True, 3, 40, 72, 12, True), (False, 3, 40, 72, 0, False), (False, 5, 33, 50, 7, True), (True, 1, 7, 1000, 3, True), (False, 16, 128, 512, 64, True)])
def test_latent_prepare(f32, H, d, r, E, gate):
    torch.manual_seed(1)
    T, ldt, tn, eps = 21, 64, 16, 1e-3
    dp, rp = -(-d // 64) * 64, -(-r // 64) * 64
    dt = torch.float32 if f32 else torch.bfloat16
    n = H * d + r + (H if gate else 0) + E
    proj = torch.randn(T, -(-n // 8) * 8, device=DEV) * 2
    nw = torch.randn(r)
    slots = torch.randperm(128)[:T]
    q, cache = torch.zeros(H * ldt, dp, dtype=dt, device=DEV), torch.full((128, rp + 64), 9.0, dtype=dt, device=DEV)
    g = torch.zeros(T, H, device=DEV) if gate else None
    lg = torch.zeros(T, E, device=DEV) if E else None
    tiles, nt = torch.zeros(H * 4, 4, dtype=torch.int32, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    ops.latent_prepare(proj, nw.to(DEV), i32(slots.tolist()), q, cache, g, lg, tiles, nt, T=T, ldt=ldt, H=H, d=d, r=r, rp=rp, E=E, tn=tn, eps=eps, status=status)
    P = proj.cpu()
    tol = 1e-6 if f32 else 4e-3
    assert rel(q.view(H, ldt, dp)[:, :T, :d], P[:, :H * d].reshape(T, H, d).transpose(0, 1)) < tol and float(q.view(H, ldt, dp)[:, :, d:].abs().sum()) == 0
    c = oracle.rms_norm(P[:, H * d:H * d + r], nw, eps)
    assert rel(cache[slots.to(DEV), :r], c) < tol and float(cache[slots.to(DEV), r:rp].abs().sum()) == 0
    assert float((cache[:, rp:] - 9).abs().sum()) == 0                                # a wider row of another layer is left alone
    if gate:
        assert torch.allclose(g.cpu(), torch.sigmoid(P[:, H * d + r:H * d + r + H]), atol=1e-6)
    if E:
        assert torch.equal(lg.cpu(), P[:, n - E:n])
    want = [[h, h * ldt + r0, min(tn, T - r0), 0] for h in range(H) for r0 in range(0, T, tn)]
    assert int(nt[0]) == len(want) and tiles[:len(want)].tolist() == want and int(status[0]) == 0


class Paged:
    """A paged latent cache with sequences on scattered pages; slots nobody owns hold large finite noise."""

    def __init__(self, lens, r, dt, row=None, seed=0, scale=1.0):
        g = torch.Generator().manual_seed(seed)
        rp = -(-r // 64) * 64
        need = [-(-n // 64) for n in lens]
        total = sum(need) + 3
        ids = (torch.randperm(total - 1, generator=g) + 1).tolist()
        self.pages = [[ids.pop() for _ in range(n)] for n in need]
        store = torch.randn(total * 64, row or rp, generator=g) * 40
        self.rows = []
        for n, pg in zip(lens, self.pages):
            c = (torch.randn(n, r, generator=g) * scale).to(dt).float()
            self.rows.append(c)
            for j in range(n):
                s = pg[j // 64] * 64 + j % 64
                store[s] = 0 if (row or rp) == rp else store[s]
                store[s, :rp] = 0
                store[s, :r] = c[j]
        self.store = store.to(dt).to(DEV)
        self.table = torch.zeros(len(lens), max(need), dtype=torch.int32)
        for i, pg in enumerate(self.pages):
            self.table[i, :len(pg)] = torch.tensor(pg)
        self.table = self.table.to(DEV)

    def tmap(self, rp):
        from cuteafd_b200.ops.native import call
        host = torch.zeros(128, dtype=torch.uint8)
        call("cuteafd_tmap_encode_latent_rows", host.data_ptr(), self.store.data_ptr(), self.store.shape[0], rp, self.store.shape[1])
        return host.to(DEV)


def attend(q, c, first, scale):
    """q [n, H, r] at positions first.. over latent rows c -> [n, H, r] attended latents."""
    s = torch.einsum("nhr,kr->nhk", q, c) * scale
    see = torch.arange(c.shape[0])[None] <= (first + torch.arange(q.shape[0]))[:, None]
    return torch.einsum("nhk,kr->nhr", torch.softmax(s.masked_fill(~see[:, None], -float("inf")), -1), c)


BORDERS = (0, 1, 62, 63, 64, 65, 127, 128, 129, 191, 192)


@pytest.mark.parametrize("H,r,splits,gate", [(3, 50, 1, True), (4, 96, 4, False), (6, 192, 3, True), (16, 256, 1, True), (1, 300, 5, True), (24, 384, 2, False),
                                             (5, 448, 1, True), (128, 512, 2, True), (40, 512, 1, False)])
def test_absorbed_attention(H, r, splits, gate):
    """Ragged batch (a prompt portion, decoded tokens, a first token) with planted keys at page borders, on scattered pages."""
    torch.manual_seed(2)
    lens, q_lens = [333, 64, 193, 1, 65], [70, 1, 2, 1, 65]
    rp, dt = -(-r // 64) * 64, torch.bfloat16
    pg = Paged(lens, r, dt, row=rp + 64)
    T, ldt = sum(q_lens), sum(q_lens) + 5
    starts = [sum(q_lens[:i]) for i in range(len(q_lens))]
    q = torch.zeros(H, ldt, rp)
    q[:, :T, :r] = torch.randn(H, T, r) * 0.2
    for s, (n, m) in enumerate(zip(lens, q_lens)):             # most rows point at one key: first, last, borders, self
        for i in range(m):
            pos = n - m + i
            for h in range(H):
                keys = [b for b in BORDERS if b <= pos] + [pos]
                key = keys[(i * 7 + h) % len(keys)]
                c = pg.rows[s][key]
                if (i + h) % 4:
                    q[h, starts[s] + i, :r] += c * (14.0 / float(c @ c))
    q = q.to(dt)
    g = torch.rand(T, H) + 0.5 if gate else None
    out = torch.full((H * ldt, rp), 7.0, dtype=dt, device=DEV)
    po = torch.full((splits * T * H * rp,), float("nan"), device=DEV) if splits > 1 else None
    pml = torch.full((splits * T * H * 2,), float("nan"), device=DEV) if splits > 1 else None
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    args = (i32(lens), i32(starts), i32(q_lens), g.to(DEV) if gate else None)
    ops.latent_attention(q.reshape(H * ldt, rp).to(DEV), pg.tmap(rp), pg.table, *args, out, T=T, ldt=ldt, n_seq=len(lens), max_q_len=max(q_lens), H=H, rank_pad=rp,
                         n_splits=splits, part_o=po, part_ml=pml, scale=0.9, status=status)
    simt = torch.zeros_like(out)
    ops.latent_attention_simt(q.reshape(H * ldt, rp).to(DEV), pg.store, pg.table, *args, simt, T=T, ldt=ldt, n_seq=len(lens), H=H, rank_pad=rp, scale=0.9, status=status)
    assert int(status[0]) == 0
    got, got2 = out.view(H, ldt, rp).float().cpu(), simt.view(H, ldt, rp).float().cpu()
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        want = attend(q[:, starts[s]:starts[s] + m, :r].float().transpose(0, 1), pg.rows[s], n - m, 0.9)
        if gate:
            want = want * g[starts[s]:starts[s] + m, :, None]
        for o in (got, got2):
            o = o[:, starts[s]:starts[s] + m].transpose(0, 1)
            err = (o[..., :r] - want).norm(dim=-1) / want.norm(dim=-1)
            assert float(err.max()) < 2e-2, (s, float(err.max()))
            assert float(o[..., r:].abs().max()) == 0 if rp > r else True
    assert float((got[:, T:] - 7).abs().max()) == 0            # rows past the step stay untouched


@pytest.mark.parametrize("H,d,dv,r,gate", [(3, 40, 24, 72, True), (2, 128, 128, 512, False), (5, 64, 65, 100, True), (4, 192, 80, 256, True), (2, 100, 100, 64, False), (1, 1, 1, 8, True)])
def test_expanding_prefill_attention(H, d, dv, r, gate):
    """Portions with a cached context in front: gather, expansion, per-head attention with planted far keys; ragged tiles."""
    from cuteafd_b200.ops.native import call, ptr, stream
    torch.manual_seed(3)
    lens, q_lens = [400, 131, 64], [200, 131, 1]
    rp, dp, dvp, dt = -(-r // 64) * 64, -(-d // 64) * 64, -(-dv // 64) * 64, torch.bfloat16
    pg = Paged(lens, r, dt, row=rp + 128, scale=1.0)
    T, ldt = sum(q_lens), sum(q_lens) + 3
    starts, ctx, tot = [0, 200, 331], [], 0
    for n in lens:
        ctx.append(tot)
        tot += -(-n // 64) * 64
    uk, uv = (torch.randn(H, d, r) * r ** -0.5).to(dt).float(), (torch.randn(H, dv, r) * r ** -0.5).to(dt).float()
    q = torch.zeros(H, ldt, dp)
    q[:, :T, :d] = torch.randn(H, T, d) * 0.3
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        for i in range(0, m, 3):
            keys = [b for b in BORDERS if b <= n - m + i]
            for h in range(H):
                k = uk[h] @ pg.rows[s][keys[(i + h) % len(keys)]]
                q[h, starts[s] + i, :d] += k * min(12.0 / float(k @ k), 20.0)
    q = q.to(dt)
    g = torch.rand(T, H) + 0.5 if gate else None
    kvw = torch.zeros(H, dp + dvp, rp)
    kvw[:, :d, :r], kvw[:, dp:dp + dv, :r] = uk, uv
    w = ops.TcWeight.from_master(kvw.reshape(H * (dp + dvp), rp), "bf16", DEV)
    cap = tot + 64
    lat, kvb = torch.zeros(cap, rp, dtype=dt, device=DEV), torch.zeros(cap, H * (dp + dvp), dtype=dt, device=DEV)
    ldo = -(-(H * dv) // 8) * 8
    out = torch.full((T, ldo), 7.0, dtype=dt, device=DEV)
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    kl, qs, ql, cs = i32(lens), i32(starts), i32(q_lens), i32(ctx)
    call("cuteafd_latent_gather_ctx", ptr(pg.store), ptr(pg.table), ptr(cs), ptr(kl), ptr(lat), 3, max(lens), pg.table.shape[1], pg.store.shape[0], cap, rp,
         pg.store.shape[1], ptr(status), stream())
    for s, n in enumerate(lens):
        assert torch.equal(lat[ctx[s]:ctx[s] + n, :r].float().cpu(), pg.rows[s])
    ops.tc_linear(w, ops.ActBuffer.wrap_bf16(lat, 256), kvb, rows=tot, status=status)
    qd, gd = q.reshape(H * ldt, dp).to(DEV), g.to(DEV) if gate else None
    call("cuteafd_latent_prefill_attention", ptr(qd), None, ptr(kvb), None, 0, 0, None, cap, ptr(cs), ptr(kl), ptr(qs), ptr(ql), ptr(gd), ptr(out), T, ldt, 3, max(q_lens), H, dp, dvp, dv,
         ldo, 0.8, ptr(status), stream())
    assert int(status[0]) == 0
    got = out.float().cpu()
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        for h in range(H):
            k, v = pg.rows[s] @ uk[h].T, pg.rows[s] @ uv[h].T
            sc = q[h, starts[s]:starts[s] + m, :d].float() @ k.T * 0.8
            see = torch.arange(n)[None] <= (n - m + torch.arange(m))[:, None]
            want = torch.softmax(sc.masked_fill(~see, -float("inf")), -1) @ v
            if gate:
                want = want * g[starts[s]:starts[s] + m, h:h + 1]
            o = got[starts[s]:starts[s] + m, h * dv:(h + 1) * dv]
            assert rel(o, want) < 2e-2 and float((o - want).abs().max()) < 0.06 * float(want.abs().max()), (s, h)
    assert float((got[:, H * dv:] - 7).abs().sum()) == 0


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("T", [5, 16, 40, 100, 300])
def test_linear_forms(kind, T):
    """Squared-ReLU epilogue over an expert tile table, token-major output of a product grouped over heads, plain fp32 output."""
    torch.manual_seed(4)
    dt = torch.float32 if kind == "f32" else torch.bfloat16
    rd = lambda *s: torch.randn(*s).to(dt).float()
    tol = 2e-6 if kind == "f32" else 6e-3
    tn = ops.pick_tn(min(T, 128))
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    G, N, K, cap = 3, 150, 72, T + 9
    w, x = rd(G, N, K), rd(G * cap, K)
    wt = ops.TcWeight.from_master(w, kind, DEV)
    act = ops.ActBuffer.alloc(wt.kind, G * cap, K, tn, DEV)
    act.data.copy_(x.to(dt))
    tiles = [[h, h * cap + r0, min(tn, T - r0), 0] for h in range(G) for r0 in range(0, T, tn)]
    tk = dict(tiles=i32(tiles), n_tiles=i32([len(tiles)]), max_tiles=len(tiles) + 2, status=status)
    y = torch.full((T, 456), 5.0, dtype=dt, device=DEV)
    ops.tc_linear(wt, act, y, rows=G * cap, token_major=(cap, 150), **tk)
    want = torch.cat([x[h * cap:h * cap + T] @ w[h].T for h in range(G)], 1)
    assert rel(y[:, :450], want) < tol and float((y[:, 450:] - 5).abs().sum()) == 0
    y2 = torch.zeros(G * cap, N, dtype=dt, device=DEV)
    ops.tc_linear(wt, act, y2, rows=G * cap, act="relu2", **tk)
    for h in range(G):
        assert rel(y2[h * cap:h * cap + T], torch.relu(x[h * cap:h * cap + T] @ w[h].T).square()) < 2 * tol
    one = ops.TcWeight.from_master(w[0], kind, DEV)
    y3 = torch.zeros(T, N + 2, device=DEV)
    ops.tc_linear(one, act, y3, rows=T, status=status)
    assert rel(y3[:, :N], x[:T] @ w[0].T) < 2e-6 and int(status[0]) == 0


@pytest.mark.parametrize("T", [3, 64, 65, 700])
def test_group_ranking_by_the_best_member(T):
    torch.manual_seed(5)
    E, k, G, keep = 24, 5, 6, 2
    z = torch.randn(T, E) * 2
    z[0] = -5.0
    z[0, [0, 8, 9, 12]] = torch.tensor([3.0, 2.0, 2.0, 2.5])      # group 2 has the best pair; by best member groups 0 and 3 stay
    idx, wts = torch.zeros(T, k, dtype=torch.int32, device=DEV), torch.zeros(T, k, device=DEV)
    ops.router_select(z.to(DEV), None, idx, wts, T, k, "softmax", True, 1.7, G, keep, group_score="max")
    idx2, wts2 = torch.zeros_like(idx), torch.zeros_like(wts)
    rows, tn = T * k, 32
    b = {n: torch.zeros(s, dtype=torch.int32, device=DEV) for n, s in dict(src=rows, slot=rows, cnt=E, off=E, tiles=(E + rows) * 4, nt=1, nr=1).items()}
    if rows <= 4096:
        ops.router_select_pack(z.to(DEV), None, idx2, wts2, T, k, "softmax", True, 1.7, G, keep, b["src"], b["slot"], b["cnt"], b["off"], b["tiles"], b["nt"], b["nr"],
                               0, E, tn, E + rows, group_score="max")
        assert torch.equal(idx, idx2) and torch.equal(wts, wts2) and int(b["nr"][0]) == rows
    want = oracle.route(z, torch.eye(E), {"experts": E, "top": k, "scale": 1.7, "groups": {"count": G, "keep": keep}})
    for t in range(T):
        got = {int(e): float(w) for e, w in zip(idx[t], wts[t])}
        assert set(got) == {e for e, _ in want[t]} and all(abs(got[e] - w) < 1e-5 for e, w in want[t]), t
    assert {0, 12} <= set(idx[0].tolist()) and not {8, 9} & set(idx[0].tolist())


# ------------------------------------------------------------------ engine
def build(cfg, tmp_path, dtype="float32", seed=0, max_tokens=2048, live=4, noise=True, tensors=None):
    from cuteafd_b200.serving.trace import TraceReplay
    t = tensors or make_tensors(cfg, seed)
    p = write_snapshot(cfg, t, tmp_path / f"{dtype}{seed}")
    rep = TraceReplay(str(p), dtype=dtype, max_tokens=max_tokens, max_live=live)
    if noise:      # what an earlier owner of a page could have left behind: large, finite
        g = torch.Generator(device=DEV).manual_seed(9)
        rep.engine.kv.normal_(0, 30, generator=g)
    return rep, t


def tokens(cfg, n, seed):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_portions(rep, rid, toks, cuts, end=True):
    """Feeds `toks` in portions of the given sizes (the last one repeats); returns logits of every position."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = cuts[min(i, len(cuts) - 1)]
        part = toks[at:at + n]
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
    else:        # a near tie of two experts may fall the other way in 16 bits: a few positions, never most
        assert float(e.median()) < 0.04 and float((e > 0.15).float().mean()) < 0.1, (float(e.median()), float(e.max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompts_portions_and_decoding_match_the_oracle(name, dtype, tmp_path):
    cfg = CONFIGS[name]
    rep, t = build(cfg, tmp_path, dtype)
    toks = tokens(cfg, 210, 1)
    want = oracle.logits(cfg, t, toks)
    rep.engine.tap = [] if dtype == "float32" else None
    whole = run_portions(rep, "a", toks, [len(toks)])
    check(whole, want, dtype)
    if dtype == "float32":
        taps, ref = rep.engine.tap, oracle.hidden_states(cfg, t, toks)
        assert len(taps) == len(ref) and all(rel(a, b) < 1e-5 for a, b in zip(taps, ref))
        rep.engine.tap = None
    for i, cuts in enumerate(([130, 1], [2, 2, 3, 57, 64, 2, 63, 2], [1], [64, 64, 1], [33])):
        got = run_portions(rep, f"p{i}", toks, cuts)
        check(got, want, dtype)
    assert rep.pool.n_free == rep.pool.n_pages - 1


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_equal_each_alone_and_pages_are_reused(dtype, tmp_path):
    cfg = MIXED
    rep, t = build(cfg, tmp_path, dtype, max_tokens=64 * 9)
    reqs = {"a": tokens(cfg, 150, 2), "b": tokens(cfg, 9, 3), "c": tokens(cfg, 70, 4), "d": tokens(cfg, 129, 5)}
    ref = {k: oracle.logits(cfg, t, v) for k, v in reqs.items()}
    got = {k: [] for k in reqs}
    at = {k: 0 for k in reqs}
    plans = [{"a": 128, "b": 1}, {"b": 1, "c": 29}, {"a": 2, "b": 1, "c": 1}, {"b": 2, "c": 3}, {"a": 1, "b": 1, "d": 61}, {"d": 3, "a": 1}, {"a": 1, "b": 1, "c": 1, "d": 1},
             {"a": 1, "b": 1, "c": 1, "d": 1}]
    for rnd in range(3):                                     # freed pages are taken again by the next pass, in another order
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
        assert rep.pool.n_free == rep.pool.n_pages - 1


def sharp(cfg, t, layer, head, key_token, query_token, strength):
    """Makes one head of one layer, at rows of `query_token`, point at rows of `key_token`: the latent rows of that token get a direction of
    their own (first embedding channel), the head's query reads the query token's channel."""
    m = cfg["layers"][layer]["mixer"]
    d = m["dim"]
    t["embed"][:, :2] = 0
    t["pos"][:, :2] = 0
    t["embed"][key_token, 0], t["embed"][query_token, 1] = 12.0, 12.0
    t[f"l{layer}.mix.dkv"][:, 1] = 0
    t[f"l{layer}.mix.dkv"][0], t[f"l{layer}.mix.dkv"][0, 0] = 0, 30.0               # latent channel 0 = "this is the key token"
    q = t[f"l{layer}.mix.q"].view(m["heads"], d, -1)
    uk = t[f"l{layer}.mix.uk"].view(m["heads"], d, -1)
    q[head, 0], uk[head, 0] = 0, 0
    q[head, 0, 1], uk[head, 0, 0] = strength, 1.0
    for k in list(t):
        t[k] = t[k].to(torch.bfloat16).float()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_keys_decide_the_output_in_prompts_and_decoding(dtype, tmp_path):
    """One score stands out among hundreds: moving the key token by one place must show, at page borders and at the very first token."""
    cfg = variant(MIXED, loop=None, layers=[MIXED["layers"][0], MIXED["layers"][3]])
    t = make_tensors(cfg, 7)
    sharp(cfg, t, 0, 1, key_token=5, query_token=6, strength=8.0)
    rep, t = build(cfg, tmp_path, dtype, tensors=t)
    for where in (0, 1, 63, 64, 127, 128, 191):
        toks = [x if x not in (5, 6) else 7 for x in tokens(cfg, 270, 8)]
        toks[where], toks[200], toks[255], toks[256], toks[269] = 5, 6, 6, 6, 6
        want = oracle.logits(cfg, t, toks)
        alone = oracle.logits(cfg, t, toks[:where] + [7] + toks[where + 1:])        # the same without the key
        for q in (200, 255, 256, 269):
            assert float(errors(alone[q:q + 1], want[q:q + 1])) > 0.2               # the planted key matters
        for cuts in ([270], [199, 1]) if where in (0, 64) else ([198, 2, 55, 1],):
            got = run_portions(rep, "x", toks, cuts)
            e = errors(got, want)[[200, 255, 256, 269]]
            assert float(e.max()) < (1e-4 if dtype == "float32" else 0.08), (where, cuts, e.tolist())


def test_first_tokens_and_single_token_prompts(tmp_path):
    for name, cfg in (("odd", ODD), ("once", ONCE)):
        rep, t = build(cfg, tmp_path / name, "float32")
        for n in (1, 2, 3):
            toks = tokens(cfg, n, 20 + n)
            check(run_portions(rep, f"r{n}", toks, [n]), oracle.logits(cfg, t, toks), "float32")


def test_long_decoding_crosses_pages_and_split_counts(tmp_path):
    cfg = variant(WIDE, layers=WIDE["layers"][:2], loop={"start": 0, "stop": 1, "times": 2})
    rep, t = build(cfg, tmp_path, "bfloat16")
    toks = tokens(cfg, 330, 30)
    want = oracle.logits(cfg, t, toks)
    got = run_portions(rep, "a", toks, [60, 1])
    check(got, want, "bfloat16")
    assert rep.engine.graph_captures >= 2                     # decode steps replay captured graphs; the split count grew with the context


def test_positions_beyond_the_table_are_refused(tmp_path):
    rep, _ = build(variant(ODD, max_positions=8), tmp_path, tensors={k: v[:8] if k == "pos" else v for k, v in make_tensors(ODD).items()})
    rep.step([{"id": "a", "tokens": [1] * 8, "want": [7]}], [])
    with pytest.raises(ValueError, match="learned positions"):
        rep.step([{"id": "a", "tokens": [1], "want": [0]}], [])


def test_greedy_generation_through_generate_and_the_scheduler(tmp_path):
    """The public generation call, and the scheduler with prefix reuse and drafts, emit the oracle's greedy tokens (fp32 engine)."""
    import argparse

    from cuteafd_b200.cli import build_serving
    from cuteafd_b200.engine.generate import BatchGenerator, generate
    from cuteafd_b200.engine.registry import build_engine, load_weights, model_spec
    from cuteafd_b200.serving.scheduler import Request
    cfg = MIXED
    t = make_tensors(cfg, 11)
    p = str(write_snapshot(cfg, t, tmp_path / "m"))
    prompts = [tokens(cfg, n, 40 + n) for n in (67, 5, 130)]
    prompts.append(prompts[2][:128] + tokens(cfg, 6, 50))     # shares two pages with the request before it
    want = [oracle.greedy(cfg, t, q, 10)[0] for q in prompts]
    spec = model_spec(p, dtype="float32")
    eng = build_engine(spec, load_weights(p, spec, torch.device(DEV)), n_pages=16, max_seqs=4, max_pages_per_seq=8)
    assert generate(eng, prompts, 10) == want
    g = BatchGenerator(eng, prefill_chunk=48)                # several chunks per prompt, none of them waiting for logits
    first = g.prefill(prompts)
    assert first == [w[0] for w in want] and g.decode_step() == [w[1] for w in want]
    ns = argparse.Namespace(model=p, device=0, dtype="float32", max_context=4096, max_sequences=4, pool_tokens=64 * 24, prefill_batch_tokens=50, decode_share=0.3,
                            prefix_cache_entries=8, prefix_cache_min_tokens=64, draft="ngram", draft_limit=3, layers=0, host_cache_gib=0.0)
    spec2, sched = build_serving(ns)
    assert spec2 == spec and sched.max_context == cfg["max_positions"]
    out = {}
    for i, q in enumerate(prompts):
        sched.submit(Request(f"r{i}", q, max_tokens=10, on_token=lambda tk, fin, why, i=i: out.setdefault(i, []).extend(tk)))
        if i == 2:
            sched.run_until_idle()                           # the third prompt's pages are in the prefix cache when the fourth arrives
    sched.run_until_idle()
    assert [out[i] for i in range(4)] == want and sched.prefix.snapshot()["hits"] >= 1


def test_trace_program_end_to_end(tmp_path):
    cfg = ONCE
    t = make_tensors(cfg, 13)
    p = write_snapshot(cfg, t, tmp_path / "m")
    a, b = tokens(cfg, 80, 60), tokens(cfg, 5, 61)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[70:], "want": [0, 9]}, {"id": "b", "tokens": b, "want": [4, 0]}], "end": ["a"]},
             {"step": 2, "entries": [], "end": ["b"]}]
    root = Path(__file__).resolve().parent.parent
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(p), "--dtype", "float32", "--out", str(out), "--max-tokens", "192"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300, env={**os.environ, "PATH": f"{Path(sys.executable).parent}:{os.environ['PATH']}"})
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    got = torch.frombuffer(bytearray((out / "1.f32").read_bytes()), dtype=torch.float32).reshape(4, cfg["vocab"])
    wa, wb = oracle.logits(cfg, t, a), oracle.logits(cfg, t, b)
    check(got, torch.stack([wa[70], wa[79], wb[4], wb[0]]), "float32")
    assert sorted(x.name for x in out.iterdir()) == ["1.f32"]

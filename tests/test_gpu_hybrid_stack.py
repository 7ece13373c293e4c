"""Hybrid recurrent / windowed-attention stacks on a GPU: every kernel of the design against plain formulas, then the engine (fp32 and bf16)
against the oracle over prompts, portions, mixed batches, decoding, reused pages and slots, drafts, the scheduler and the trace program."""
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from hybrid_stack_models import CONFIGS, MIXED, PLAIN, attention, make_tensors, rglru, variant, write_snapshot, yarn
from stack_helpers import DEPTH, DEV, STEPS, Paged, i32, meta, rel, status_word

from cuteafd_b200 import ops
from cuteafd_b200.ref import hybrid_stack as oracle

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ kernels
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("W", [40, 1283, 9000])
def test_norm_rows(W, f32):
    torch.manual_seed(0)
    T, V, Wp, eps = 37, 50, -(-W // 8) * 8, 0.3
    dt, tol = (torch.float32, 2e-6) if f32 else (torch.bfloat16, 4e-3)
    pad = lambda t: torch.nn.functional.pad(t, (0, Wp - W)).to(DEV)
    table, toks = torch.randn(V, W).to(torch.bfloat16), torch.randint(0, V, (T,))
    g1, g2, gp, bias = (torch.randn(W) for _ in range(4))
    x, xn, st = torch.zeros(T, Wp, device=DEV), torch.full((T, Wp + 8), 5.0, dtype=dt, device=DEV), status_word()
    kw = dict(f32=f32, eps=eps, status=st)
    ops.norm_rows(x, W, T, tokens=i32(toks.tolist()), table=pad(table), gain=pad(g1), xn=xn, **kw)
    want = table.float()[toks]
    assert torch.equal(x[:, :W].cpu(), want) and rel(xn[:, :W], oracle.rms_norm(want, g1, eps)) < tol and float((xn[:, Wp:] - 5).abs().sum()) == 0
    add = torch.randn(T, W).to(dt)
    ops.norm_rows(x, W, T, add=pad(add), bias=pad(bias), post=pad(gp), mult=0.37, gain=pad(g2), xn=xn, **kw)
    want = want + 0.37 * oracle.rms_norm(add.float() + bias, gp, eps)
    assert rel(x[:, :W], want) < 2e-6 and rel(xn[:, :W], oracle.rms_norm(want, g2, eps)) < tol
    ops.norm_rows(x, W, T, add=pad(add), mult=-1.5, **kw)                      # no norm behind, nothing for a next product
    want = want - 1.5 * add.float()
    assert rel(x[:, :W], want) < 2e-6
    rows = [5, 0, 36, 5]
    out = torch.zeros(4, Wp, dtype=dt, device=DEV)
    ops.norm_rows(x, W, 4, src_rows=i32(rows), gain=pad(g1), xn=out, **kw)
    assert rel(out[:, :W], oracle.rms_norm(want[rows], g1, eps)) < tol and float(out[:, W:].abs().sum()) == 0 and int(st[0]) == 0
    ops.norm_rows(x, W, 1, tokens=i32([V]), table=pad(table), **kw)            # a token outside the table is reported, not read
    assert int(st[0]) >> 24 == 5


@pytest.mark.parametrize("rot", [{"dims": 12, "base": 10000.0, "scaling": yarn(4.0, 64)}, {"dims": 2, "base": 500.0, "scaling": None}, {"dims": 256, "base": 1e6, "scaling": yarn(40.0, 4096, 32.0)}])
def test_rope_table_at_near_and_far_positions(rot):
    from cuteafd_b200.config import AttentionSpec, RopeScaling
    from cuteafd_b200.models.hybrid_stack import rope_frequencies
    sc = rot["scaling"]
    a = AttentionSpec(rope_dims=rot["dims"], rope_theta=rot["base"], rope_scaling=RopeScaling(**sc) if sc else None)
    f, amp = rope_frequencies(a)
    f = torch.tensor(f, dtype=torch.float64)
    pos = [0, 1, 2, 63, 64, 1000, 70001, 1000003]
    out = torch.zeros(len(pos), len(f), 2, device=DEV)
    ops.rope_table(i32(pos), torch.stack([f.float(), (f - f.float().double()).float()]).to(DEV), amp, out, len(pos))
    want, wamp = oracle.rope_frequencies(rot)
    ang = torch.tensor(pos, dtype=torch.float64)[:, None] * torch.tensor(want, dtype=torch.float64)
    assert float((out.double().cpu() - torch.stack([ang.cos(), ang.sin()], -1) * wamp).abs().max()) < 1e-6


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dim,vdim,taps,rot", [(3, 1, 40, 24, 3, 12), (7, 7, 33, 45, 5, 10), (4, 2, 128, 128, 4, 128), (2, 1, 256, 200, 2, 64), (5, 0, 72, 136, 1, 72), (1, 1, 2, 1, 16, 2)])
def test_conv_qkv_across_portions(H, G, dim, vdim, taps, rot, f32):
    """Convolution, head norms and rotation of every portion equal those of the whole sequence, wherever it is cut and after steps back."""
    torch.manual_seed(1)
    dt, tol, eps = (torch.float32, 3e-6, 1e-3) if f32 else (torch.bfloat16, 6e-3, 1e-3)
    up = lambda n: -(-n // 64) * 64
    dp, dvp, C = up(dim), up(vdim), (H + G) * dim + G * vdim
    sp = {"dims": rot, "base": 300.0, "scaling": yarn(3.0, 50)}
    slots, L = [2, 0, 3], 240
    u = [torch.randn(L, C).to(dt).float() for _ in slots]
    w, qn, kn = torch.randn(C, taps), torch.randn(dim), torch.randn(dim)
    want = []
    for x in u:
        y = oracle.causal_conv(x, w)
        q = oracle.rotate(oracle.rms_norm(y[:, :H * dim].reshape(L, H, dim), qn, eps), sp)
        k = oracle.rotate(oracle.rms_norm(y[:, H * dim:(H + G) * dim].reshape(L, G, dim), kn, eps), sp) if G else torch.zeros(L, 0, dim)
        want.append((q, k, y[:, (H + G) * dim:].reshape(L, G, vdim)))
    freq, amp = oracle.rope_frequencies(sp)
    f = torch.tensor(freq, dtype=torch.float64)
    freq = torch.stack([f.float(), (f - f.float().double()).float()]).to(DEV)
    ring = torch.full((4, taps - 1 + DEPTH, C), 50.0, dtype=dt, device=DEV)                     # what another sequence left behind
    cache = torch.full((700, max(8, G * (dp + dvp)) + 64), 9.0, dtype=dt, device=DEV)
    st = status_word()
    for runs in STEPS:
        T = sum(n for _, n in runs)
        where = torch.randperm(700, generator=torch.Generator().manual_seed(T))[:T].tolist()
        md = meta(runs, slots, where)
        proj = torch.full((T, -(-C // 8) * 8), 77.0, dtype=dt, device=DEV)
        proj[:, :C] = torch.cat([u[s][p:p + n] for s, (p, n) in enumerate(runs)]).to(dt)
        table = torch.zeros(T, rot // 2, 2, device=DEV)
        ops.rope_table(i32([p + i for p, n in runs for i in range(n)]), freq, amp, table, T)
        q = torch.zeros(T, H * dp, dtype=dt, device=DEV)
        for rep in range(2 if max(n for _, n in runs) <= DEPTH else 1):                         # a repeated short step changes nothing
            ops.conv_qkv(proj, w.T.contiguous().to(DEV), qn.to(DEV), kn.to(DEV), table, ring, q, cache, md, H=H, G=G, dim=dim, dp=dp, vdim=vdim, dvp=dvp, pairs=rot // 2,
                         eps=eps, n_seq=len(runs), max_q_len=max(n for _, n in runs), status=st)
        assert int(st[0]) == 0
        row = 0
        for s, (p, n) in enumerate(runs):
            got = q[row:row + n].view(n, H, dp)
            assert rel(got[..., :dim], want[s][0][p:p + n]) < tol and float(got[..., dim:].abs().sum()) == 0, runs
            if G:
                c = cache[torch.tensor(where[row:row + n], device=DEV)]
                assert rel(c[:, :G * dp].view(n, G, dp)[..., :dim], want[s][1][p:p + n]) < tol, runs
                assert rel(c[:, G * dp:G * (dp + dvp)].view(n, G, dvp)[..., :vdim], want[s][2][p:p + n]) < tol, runs
                assert float((c[:, G * (dp + dvp):] - 9).abs().sum()) == 0                      # a wider row of another layer is left alone
            row += n


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("C,blocks,taps", [(120, 3, 3), (45, 3, 1), (35, 1, 6), (512, 2, 4), (128, 32, 2), (70, 5, 16)])
def test_recurrence_across_portions(C, blocks, taps, f32):
    """Convolution, block gates, recurrence and GELU branch of every portion equal those of the whole sequence; channels with long memories carry
    their state through every kind of portion."""
    torch.manual_seed(2)
    dt, tol = (torch.float32, 5e-6) if f32 else (torch.bfloat16, 8e-3)
    up = lambda n: -(-n // 8) * 8
    sq, n8, L, slots = C // blocks, up(C), 240, [1, 3, 0]
    rd = lambda *s, std=1.0: (torch.randn(*s) * std).to(dt).float()
    xb, yb, cb, w = torch.randn(C) * 0.3, torch.randn(C) * 0.3, torch.randn(C) * 0.3, torch.randn(C, taps) * 0.6
    ra, ri = rd(blocks, sq, sq, std=sq ** -0.5), rd(blocks, sq, sq, std=sq ** -0.5)
    rb, ib, lam = torch.randn(blocks, sq) - 2.0, torch.randn(blocks, sq), torch.randn(C) * 2 - 3.0
    lam[0] = -9.0                                                                              # forgets nothing for thousands of tokens
    x, y = [rd(L, C) for _ in slots], [rd(L, C) for _ in slots]
    want, conv = [], []
    for xs, ys in zip(x, y):
        u = oracle.causal_conv(xs + xb, w, cb)
        conv.append(u)
        u = u.to(dt).float()
        s = oracle.lru(u.double(), oracle.block_gate(u, ra, rb).double(), oracle.block_gate(u, ri, ib).double(), lam.double()).float()
        want.append(s * oracle.gelu_tanh(ys + yb))
    assert all(float(abs(v[200, 0])) > 0 for v in want)
    dev = lambda t: t.float().reshape(-1).to(DEV).contiguous()
    wg = ops.TcWeight.from_master(torch.nn.functional.pad(torch.cat([ra, ri], 1), (0, up(sq) - sq)), "f32" if f32 else "bf16", DEV)
    gb = dev(torch.cat([rb, ib], 1))
    decay = dev(-8.0 * torch.nn.functional.softplus(lam.double()))
    args = (dev(xb), dev(yb), w.T.contiguous().to(DEV), dev(cb))
    ring = torch.full((4, taps - 1 + DEPTH, C), 50.0, dtype=dt, device=DEV)
    state = torch.full((4, DEPTH + 1, C), 50.0, device=DEV)
    st, cap = status_word(), 256
    tn = 32
    act = ops.ActBuffer.alloc(wg.kind, blocks * cap, up(sq), tn, DEV)
    gates, out = torch.zeros(cap, 2 * C, device=DEV), torch.zeros(cap, n8, dtype=dt, device=DEV)
    tiles, nt = torch.zeros(blocks * (cap // tn), 4, dtype=torch.int32, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    agg = torch.full((cap // 64 + 5, C, 2), float("nan"), device=DEV)
    for runs in STEPS:
        T, longest = sum(n for _, n in runs), max(n for _, n in runs)
        proj = torch.full((T, 2 * n8), 77.0, dtype=dt, device=DEV)
        for o, src in ((0, y), (n8, x)):
            proj[:, o:o + C] = torch.cat([src[s][p:p + n] for s, (p, n) in enumerate(runs)]).to(dt)
        a = ops.recurrence_arg(proj[:, n8:], proj, args[0], args[1], args[2], args[3], ring, state, act.data, gates, gb, decay, agg, out, meta(runs, slots), blocks=blocks, T=T,
                               ldt=cap, tiles=tiles, n_tiles=nt, tn=tn, n_seq=len(runs), max_q_len=longest, status=st)
        for rep in range(2 if longest <= DEPTH else 1):
            ops.rglru_conv(a, f32=f32)
            ops.tc_linear(wg, act, gates, rows=blocks * cap, tiles=tiles, n_tiles=nt, max_tiles=blocks * -(-T // tn), token_major=(cap, 2 * sq), status=st)
            ops.lru_scan(a, f32=f32)
        assert int(st[0]) == 0
        row = 0
        for s, (p, n) in enumerate(runs):
            got_u = act.data.view(blocks, cap, -1)[:, row:row + n, :sq].transpose(0, 1).reshape(n, C)
            assert rel(got_u, conv[s][p:p + n]) < tol, runs
            err = (out[row:row + n, :C].float().cpu() - want[s][p:p + n]).norm(dim=-1) / want[s].norm(dim=-1).mean()
            assert float(err.max()) < 3 * tol, (runs, s, float(err.max()))
            row += n
        assert float(out[:, C:].abs().sum()) == 0


@pytest.mark.parametrize("T", [5, 16, 40, 100, 300])
def test_glu_and_softcap_epilogues(T):
    torch.manual_seed(4)
    K, N, limit, cap, st = 136, 200, 0.9, 1.5, status_word()
    rd = lambda *s: torch.randn(*s).to(torch.bfloat16).float()
    wg, wu, x, bg, bu = rd(N, K) / 8, rd(N, K) / 8, rd(T, K), torch.randn(N) * 0.3, torch.randn(N) * 0.3
    g, u = x @ wg.T, x @ wu.T
    want = oracle.clamped_glu(g + bg, u + bu, limit)
    assert float((g + bg > limit).float().mean()) > 0.1 and float(((u + bu).abs() > limit).float().mean()) > 0.1
    tn = ops.pick_tn(min(T, 128))
    act = ops.ActBuffer.alloc(ops.KIND_BF16, T, K, tn, DEV)
    act.data.copy_(x)
    W = lambda t, kind="bf16": ops.TcWeight.from_master(t, kind, DEV)
    for ldy in (N, N + 3):                                   # rows that allow 16-byte stores, and rows that do not
        y = torch.full((T, ldy), 5.0, dtype=torch.bfloat16, device=DEV)
        ops.tc_linear(W(wg), act, y, rows=T, w_up=W(wu), act="clamped_glu", bound=limit, biases=(bg.to(DEV), bu.to(DEV)), status=st)
        assert rel(y[:, :N], want) < 6e-3 and float((y[:, N:] - 5).abs().sum()) == 0
    z = torch.zeros(T, N, device=DEV)
    ops.tc_linear(W(wg), act, z, rows=T, act="softcap", bound=cap, status=st)
    assert float((z.cpu() - oracle.softcap(g, cap)).abs().max()) < 1e-5
    a32 = ops.ActBuffer.alloc(ops.KIND_F32, T, K, tn, DEV)
    a32.data.copy_(x)
    ops.tc_linear(W(wg, "f32"), a32, z, rows=T, act="softcap", bound=cap)
    assert float((z.cpu() - oracle.softcap(g, cap)).abs().max()) < 1e-5
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 6e-3)):
        out = torch.zeros(T, N, dtype=dt, device=DEV)
        ops.glu_rows(g.to(dt).to(DEV), u.to(dt).to(DEV), bg.to(DEV), bu.to(DEV), out, T, limit)
        assert rel(out, oracle.clamped_glu(g.to(dt).float() + bg, u.to(dt).float() + bu, limit)) < tol
    assert int(st[0]) == 0


@pytest.mark.parametrize("H,G,dim,vdim,window,splits", [(10, 1, 128, 72, 90, 2), (3, 3, 40, 24, 1, 1), (6, 2, 64, 64, 64, 3), (9, 1, 200, 256, 65, 1), (5, 1, 192, 33, 63, 4), (40, 1, 100, 192, 130, 1),
                                                        (12, 4, 256, 128, 0, 5), (128, 1, 16, 48, 200, 2), (4, 2, 130, 136, 4096, 7), (96, 1, 64, 130, 70, 1)])
def test_window_attention(H, G, dim, vdim, window, splits):
    """Ragged batch (prompt portions, decoded tokens, a first token) on scattered pages; rows point at the first key of their window, at the one
    just in front of it, at page borders and at themselves - the tcgen05 kernels and the ordinary-core one."""
    torch.manual_seed(5)
    lens, q_lens = [333, 64, 193, 1, 65], [130, 1, 2, 1, 65]
    dt, scale = torch.bfloat16, 0.7
    pg = Paged(lens, G, dim, vdim, dt)
    T, group = sum(q_lens), H // G
    starts = [sum(q_lens[:i]) for i in range(len(q_lens))]
    q = torch.zeros(T, H, pg.dp)
    q[..., :dim] = torch.randn(T, H, dim) * 0.1
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        for i in range(m):
            pos = n - m + i
            w = window or n
            keys = [k for k in (pos - w + 1, pos - w, pos - w + 2, pos - w - 1, 0, 63, 64, pos, pos - 1) if 0 <= k <= pos]
            for h in range(H):
                if (i + h) % 5:
                    k = pg.k[s][keys[(i * 3 + h) % len(keys)], h // group]
                    q[starts[s] + i, h, :dim] += k * (14.0 / float(k @ k))
    q = q.to(dt)
    qd = q.reshape(T, -1).to(DEV)
    ldo = -(-(H * vdim) // 8) * 8
    st = status_word()
    outs = {}
    kw = dict(T=T, n_seq=len(lens), Hq=H, Hkv=G, dp=pg.dp, dvp=pg.dvp, dv=vdim, window=window, scale=scale, status=st)
    where = (pg.table, i32(lens), i32(starts), i32(q_lens))
    maps = ops.encode_window_maps(pg.store, G, pg.dp, pg.dvp)
    new = lambda: torch.full((T, ldo), 7.0, dtype=dt, device=DEV)
    outs["simt"] = new()
    ops.window_attention_simt(qd, pg.store, *where, outs["simt"], **kw)
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
        want = oracle.attend(full, pg.k[s], pg.v[s], scale, window or None)[n - m:]
        for name, o in outs.items():
            o = o[starts[s]:starts[s] + m].float().cpu()
            err = (o[:, :H * vdim].reshape(m, H, vdim) - want).norm(dim=-1) / want.norm(dim=-1)
            assert float(err.max()) < 2e-2, (name, s, float(err.max()))
            assert float((o[:, H * vdim:] - 7).abs().sum()) == 0


# ------------------------------------------------------------------ engine
def wide(t):
    """The tensors in float64: where decays are close to one, 1 - a^2 would cost an fp32 oracle four digits."""
    return {k: v.double() for k, v in t.items()}


def logits(cfg, t, toks):
    return oracle.logits(cfg, wide(t), toks).float()


def build(cfg, tmp_path, dtype="float32", seed=0, max_tokens=2048, live=4, noise=True, tensors=None):
    from cuteafd_b200.serving.trace import TraceReplay
    t = tensors or make_tensors(cfg, seed)
    p = write_snapshot(cfg, t, tmp_path / f"{dtype}{seed}")
    rep = TraceReplay(str(p), dtype=dtype, max_tokens=max_tokens, max_live=live)
    if noise:      # what earlier owners of a page or a state slot could have left behind: large, finite
        g = torch.Generator(device=DEV).manual_seed(9)
        for buf in [rep.engine.kv] + rep.engine.rings + [s for s in rep.engine.states if s is not None]:
            buf.normal_(0, 30, generator=g)
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
    assert float(e.max()) < (5e-5 if dtype == "float32" else 0.06), float(e.max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompts_portions_and_decoding_match_the_oracle(name, dtype, tmp_path):
    cfg = CONFIGS[name]
    rep, t = build(cfg, tmp_path, dtype)
    toks = tokens(cfg, 290, 1)
    want = logits(cfg, t, toks)
    rep.engine.tap = [] if dtype == "float32" else None
    check(run_portions(rep, "a", toks, [len(toks)]), want, dtype)
    if dtype == "float32":
        taps, ref = rep.engine.tap, [x.float() for x in oracle.hidden_states(cfg, wide(t), toks)]
        assert len(taps) == len(ref) and all(rel(a, b) < 1e-5 for a, b in zip(taps, ref))
        rep.engine.tap = None
    for i, cuts in enumerate(([200, 1], [2, 2, 3, 57, 64, 2, 63, 2, 9, 8, 7, 1, 65], [1], [64, 64, 1], [33], [130, 130, 2])):
        check(run_portions(rep, f"p{i}", toks, cuts), want, dtype)
    assert rep.pool.n_free == rep.pool.n_pages - 1 and len(rep.runner._free_slots) == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_equal_each_alone_and_pages_and_slots_are_reused(dtype, tmp_path):
    cfg = MIXED
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


def sharp(cfg, t, layer, head, key_token, query_token, strength):
    """Makes one head of one attention layer, at rows of `query_token`, point at rows of `key_token`: the last (unrotated) dimension of the head
    reads a channel only these tokens have."""
    m = cfg["layers"][layer]["mixer"]
    d, kh = m["dim"], head // (m["heads"] // m["kv_heads"])
    t["embed"][:, :2] = 0
    t["embed"][key_token, 0], t["embed"][query_token, 1] = 3.0, 3.0
    p = f"l{layer}.mix"
    t[f"l{layer}.norm1"][:2] = 0
    for k, row, ch in (("q", head * d + d - 1, 1), ("k", kh * d + d - 1, 0)):
        t[f"{p}.{k}"][:, :2] = 0
        t[f"{p}.{k}"][row] = 0
        t[f"{p}.{k}"][row, ch] = 60.0
        t[f"{p}.{k}.conv"][row] = 0
        t[f"{p}.{k}.conv"][row, -1] = 1.0
        t[f"{p}.{k}.norm"][-1] = strength
    for k in list(t):
        t[k] = t[k].to(torch.bfloat16).float()


WINDOW = 100


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shared", [False, True])
def test_keys_at_the_edge_of_the_window_decide_the_output(shared, dtype, tmp_path):
    """One score stands out: the key that is just inside the window must count, the one just outside must not - in prompts, portions and decoding,
    with the layer's own keys and with another layer's, whose window is wider."""
    first = attention(2, 1, 40, 24, 400 if shared else WINDOW, 3, 12, 0.3, scaling=yarn(4.0, 64))
    layers = [first] + ([attention(4, 1, 40, 24, WINDOW, 2, 12, 0.3, scaling=yarn(4.0, 64), kv_from=0)] if shared else [])
    cfg = variant(PLAIN, layers=layers, width=96, vocab=61)
    t = make_tensors(cfg, 7)
    t["embed"][5], t["embed"][7] = torch.roll(t["embed"][7], 11), t["embed"][7]
    sharp(cfg, t, 0, 1, key_token=5, query_token=6, strength=2.2)
    if shared:          # the first layer's own queries stay flat; the second layer's point at the key
        t["l0.mix.q.norm"][-1] = 0.1
        t["l1.norm1"][:2] = 0
        t["l1.mix.q"][:, :2] = 0
        t["l1.mix.q"][3 * 40 + 39] = 0
        t["l1.mix.q"][3 * 40 + 39, 1], t["l1.mix.q.norm"][-1] = 60.0, 2.2
        t["l1.mix.q.conv"][3 * 40 + 39] = torch.tensor([0.0, 1.0])
        t["l0.norm1b"][:2] = -1.0                            # nothing is added to the two marker channels
        t = {k: v.to(torch.bfloat16).float() for k, v in t.items()}
    rep, t = build(cfg, tmp_path, dtype, tensors=t)
    n = 320
    for q in (WINDOW - 1, WINDOW, 191, 192, 255, 256, 318):
        base = [x if x not in (5, 6) else 7 for x in tokens(cfg, n, 8)]
        base[q] = 6
        for back, inside in ((WINDOW - 1, True), (WINDOW, False), (0, True), (WINDOW - 2, True), (WINDOW + 1, False)):
            k = q - back
            if k < 0 or k == q:
                continue
            toks = list(base)
            toks[k] = 5
            want, alone = logits(cfg, t, toks), logits(cfg, t, base)
            moved = float(errors(alone[q:q + 1], want[q:q + 1]))
            # (a little of the token reaches its neighbours through the convolutions, and a wider layer below)
            assert moved > 0.15 if inside else (shared or moved < 0.1), (q, back, moved)
            for cuts in ([n], [q, 1, 2]) if back in (WINDOW - 1, WINDOW) else ([q - 1, 2],):
                got = run_portions(rep, "x", toks, cuts)
                e = float(errors(got[q:q + 1], want[q:q + 1]))
                assert e < (5e-5 if dtype == "float32" else 0.03), (q, back, cuts, e)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_token_is_remembered_for_hundreds_of_tokens(dtype, tmp_path):
    """A recurrence that forgets nothing: the first token still shows at the end, through whole prompts, portions and decoding; a state that is
    lost or taken from another slot would too."""
    cfg = variant(PLAIN, layers=[rglru(64, 4, 3), rglru(48, 1, 2, ff=40)], vocab=61)
    t = make_tensors(cfg, 17)
    for p in ("l0", "l1"):
        t[f"{p}.mix.lam"][:] = -9.0
        t[f"{p}.mix.ra.b"][:] = -3.0
    t["embed"][:, 0], t["embed"][5], t["l0.norm1"][0] = 0.0, 0.0, 0.0
    t["embed"][5, 0] = 3.0                                    # its own channel, which only the x branch of the first layer reads, strongly
    t["l0.mix.x"][:, 0] = torch.randn(64, generator=torch.Generator().manual_seed(3)) * 4.0
    rep, t = build(cfg, tmp_path, dtype, tensors={k: v.to(torch.bfloat16).float() for k, v in t.items()})
    toks = [x if x != 5 else 7 for x in tokens(cfg, 400, 18)]
    other = [5] + toks[1:]
    want, with5 = logits(cfg, t, toks), logits(cfg, t, other)
    assert float(errors(with5[380:], want[380:]).min()) > 0.05
    for cuts in ([400], [390, 1], [63, 2, 64, 65, 1, 128, 9, 8, 60], [100, 100]):
        a, b = run_portions(rep, "a", toks, cuts, end=False), run_portions(rep, "b", other, cuts, end=False)
        check(a, want, dtype)
        check(b, with5, dtype)
        rep.step([], ["a", "b"])


def test_first_tokens_and_single_token_prompts(tmp_path):
    for name in ("odd", "plain", "mixed", "recurrent"):
        rep, t = build(CONFIGS[name], tmp_path / name, "float32")
        for n in (1, 2, 3):
            toks = tokens(CONFIGS[name], n, 20 + n)
            check(run_portions(rep, f"r{n}", toks, [n]), logits(CONFIGS[name], t, toks), "float32")


@pytest.mark.parametrize("name", ["wide", "mixed"])
def test_long_decoding_crosses_pages_windows_and_split_counts(name, tmp_path):
    cfg = CONFIGS[name]
    rep, t = build(cfg, tmp_path, "bfloat16")
    toks = tokens(cfg, 330, 30)
    check(run_portions(rep, "a", toks, [40, 1]), logits(cfg, t, toks), "bfloat16")
    assert rep.engine.graph_captures >= 1                     # decode steps replay captured graphs


def test_tokens_can_be_taken_back(tmp_path):
    """A step of up to `state_depth` rows may be continued from any of its rows: rejected rows leave no trace, and a repeated step none either."""
    from cuteafd_b200.engine.kv import SeqKV
    from cuteafd_b200.serving.scheduler import Request, Row, SeqState
    cfg = MIXED
    rep, t = build(cfg, tmp_path)
    toks, wrong = tokens(cfg, 120, 31), tokens(cfg, 120, 32)
    want = logits(cfg, t, toks)
    st = SeqState(Request("a", list(toks)), SeqKV())
    run = lambda tk, pos: (rep.runner.run([Row(st, tk, pos, list(range(len(tk))))]), rep.runner.last_lane.logits[:len(tk)].cpu())[1]
    check(run(toks[:71], 0), want[:71], "float32")
    pos = 71
    for keep, drafted in ((3, 8), (1, 2), (7, 8), (8, 8), (1, 8), (2, 5), (4, 7), (1, 1), (5, 8)):
        rows = toks[pos:pos + keep] + wrong[pos + keep:pos + drafted]
        check(run(rows, pos)[:keep], want[pos:pos + keep], "float32")
        pos += keep
    check(run(toks[pos:pos + 20], pos), want[pos:pos + 20], "float32")
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
    cfg = MIXED
    t = make_tensors(cfg, 11)
    p = str(write_snapshot(cfg, t, tmp_path / "m"))
    prompts = [tokens(cfg, n, 40 + n) for n in (67, 5, 130)]
    prompts.append([3, 1, 4, 1, 5] * 9)                       # repeats itself: the n-gram drafter has something to propose
    want = [oracle.greedy(cfg, wide(t), q, 14)[0] for q in prompts]
    spec = model_spec(p, dtype="float32")
    eng = build_engine(spec, load_weights(p, spec, torch.device(DEV)), n_pages=16, max_seqs=4, max_pages_per_seq=8)
    assert generate(eng, prompts, 14) == want
    assert generate(eng, prompts[::-1], 14) == want[::-1]    # pages and state slots of the first call are used again
    g = BatchGenerator(eng, prefill_chunk=48)                # several chunks per prompt, none of them waiting for logits
    first = g.prefill(prompts)
    assert first == [w[0] for w in want] and g.decode_step() == [w[1] for w in want]
    ns = argparse.Namespace(model=p, device=0, dtype="float32", max_context=4096, max_sequences=3, pool_tokens=64 * 24, prefill_batch_tokens=50, decode_share=0.3,
                            prefix_cache_entries=8, prefix_cache_min_tokens=64, draft="ngram", draft_limit=12, layers=0, host_cache_gib=0.0)
    spec2, sched = build_serving(ns)
    assert spec2 == spec and sched.prefix is None and sched.max_draft == 7
    out = {}
    for i, q in enumerate(prompts):
        sched.submit(Request(f"r{i}", q, max_tokens=14, on_token=lambda tk, fin, why, i=i: out.setdefault(i, []).extend(tk)))
    sched.run_until_idle()
    assert [out[i] for i in range(4)] == want and sched.stats["drafted"] > 0


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


def test_a_capture_survives_garbage_from_an_engine_that_is_gone(tmp_path):
    """Captured graphs of a dropped engine sit in reference cycles; the collector must not release them in the middle of another capture."""
    import gc
    toks = tokens(PLAIN, 12, 70)
    old, _ = build(PLAIN, tmp_path / "a", "bfloat16")
    for n in (1, 2, 3):
        run_portions(old, f"r{n}", toks, [n])
    assert old.engine.graph_captures >= 3
    rep, t = build(PLAIN, tmp_path / "b", "bfloat16")
    run_portions(rep, "warm", toks, [12])
    before = gc.get_threshold()
    try:
        old.engine.self_reference = old.engine
        del old
        gc.set_threshold(1, 1, 1)                            # collect at every opportunity
        check(run_portions(rep, "x", toks, [1]), logits(PLAIN, t, toks), "bfloat16")
    finally:
        gc.set_threshold(*before)
    assert rep.engine.graph_captures >= 1

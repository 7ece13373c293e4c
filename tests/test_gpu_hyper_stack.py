"""Hyper-connected stacks on a GPU: every kernel of the design against plain formulas, then the engine (fp32 and bf16) against the oracle over
prompts, portions, mixed batches, decoding, reused pages and slots, drafts, the scheduler and the trace program."""
import copy
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from hyper_stack_models import CONFIGS, MIXED, PLAIN, RANK, attn, gla, make_tensors, parallel, parallel2, plain, retention, variant, write_snapshot
from stack_helpers import DEPTH, DEV, STEPS, Paged, i32, meta, rel, status_word

from cuteafd_b200 import ops
from cuteafd_b200.ref import hyper_stack as oracle
from cuteafd_b200.ref.hybrid_stack import causal_conv, rms_norm

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------ kernels
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("S,W", [(1, 40), (2, 1283), (3, 520), (4, 9000), (5, 90), (8, 136)])
def test_stream_boundaries(S, W, f32):
    torch.manual_seed(0)
    T, V, Wp, eps = 23, 50, -(-W // 8) * 8, 0.3
    dt, tol = (torch.float32, 3e-6) if f32 else (torch.bfloat16, 4e-3)
    pad = lambda t: torch.nn.functional.pad(t, (0, Wp - W)).to(DEV).contiguous()
    dev = lambda t: t.to(DEV).contiguous()
    table, toks = torch.randn(V, W).to(torch.bfloat16), torch.randint(0, V, (T,))
    ins, outs, mixes, gains = torch.randn(3, S), torch.randn(2, S), torch.randn(2, S, S), [torch.randn(W) for _ in range(5)]
    x, xn, st = torch.full((T, S, Wp), 3.0, device=DEV), torch.full((T, Wp + 8), 5.0, dtype=dt, device=DEV), status_word()
    kw = dict(f32=f32, eps=eps, status=st)
    ops.hyper_rows(x, W, T, tokens=i32(toks.tolist()), table=pad(table), next_in=dev(ins[0]), gain=pad(gains[0]), xn=xn, **kw)
    want = [table.float()[toks]] * S
    check = lambda w: rel(x[..., :W], torch.stack(w, 1)) < 3e-6 and float(x[..., W:].abs().sum()) == 0
    assert check(want) and rel(xn[:, :W], rms_norm(oracle.collapse(want, ins[0]), gains[0], eps)) < tol and float((xn[:, Wp:] - 5).abs().sum()) == 0
    # a biased output and routed rows on top (more routes than one batch of them)
    k, n = 11, 40
    a, y, bias = torch.randn(T, W).to(dt), torch.randn(n, W).to(dt), torch.randn(W)
    slot, wts = torch.randint(0, n, (T, k)), torch.rand(T, k)
    ops.hyper_rows(x, W, T, out=dev(outs[0]), mix=dev(mixes[0]), a=pad(a), bias=pad(bias), routed=(pad(y), i32(slot.tolist()), dev(wts), k), next_in=dev(ins[1]), gain=pad(gains[1]), xn=xn, **kw)
    want = oracle.spread(want, mixes[0], outs[0], a.float() + bias + (wts[:, :, None] * y.float()[slot]).sum(1))
    assert check(want) and rel(xn[:, :W], rms_norm(oracle.collapse(want, ins[1]), gains[1], eps)) < tol
    # two outputs, each behind its own norm; nothing for a next product
    b, before = torch.randn(T, W).to(dt), xn.clone()
    ops.hyper_rows(x, W, T, out=dev(outs[1]), mix=dev(mixes[1]), a=pad(a), b=pad(b), norms=(pad(gains[2]), pad(gains[3])), scales=(0.5, 0.25), **kw)
    want = oracle.spread(want, mixes[1], outs[1], 0.5 * rms_norm(a.float(), gains[2], eps) + 0.25 * rms_norm(b.float(), gains[3], eps))
    assert check(want) and torch.equal(xn, before)
    ops.hyper_rows(x, W, T, out=dev(outs[0]), mix=dev(mixes[0]), routed=(pad(y), i32(slot[:, :2].tolist()), dev(wts[:, :2]), 2), **kw)          # routed rows alone
    want = oracle.spread(want, mixes[0], outs[0], (wts[:, :2, None] * y.float()[slot[:, :2]]).sum(1))
    assert check(want)
    rows, out = [5, 0, T - 1, 5], torch.zeros(4, Wp, dtype=dt, device=DEV)
    ops.hyper_rows(x, W, 4, src_rows=i32(rows), gain=pad(gains[4]), xn=out, **kw)
    assert rel(out[:, :W], rms_norm(sum(want)[rows], gains[4], eps)) < tol and float(out[:, W:].abs().sum()) == 0 and int(st[0]) == 0
    ops.hyper_rows(x, W, 1, tokens=i32([V]), table=pad(table), next_in=dev(ins[0]), **kw)          # a token outside the table is reported, not read
    assert int(st[0]) >> 24 == 5


@pytest.mark.parametrize("spec", [{"buckets": 97, "mul_prev": 13, "mul_cur": 7}, {"buckets": 509, "mul_prev": 100003, "mul_cur": 99991}, {"buckets": 1, "mul_prev": 2, "mul_cur": 3}])
def test_pair_rows_across_portions(spec):
    torch.manual_seed(1)
    W, V, slots, L = 48, 70000, [2, 0, 3], 240
    table, pairs = torch.randn(V, W).to(torch.bfloat16), torch.randn(spec["buckets"] + 1, W).to(torch.bfloat16)
    toks = [torch.randint(0, V, (L,)).tolist() for _ in slots]
    want = [table.float()[t] + pairs.float()[oracle.bigram_rows(t, spec)] for t in toks]
    recent, st = torch.full((4, DEPTH + 1), 77, dtype=torch.int32, device=DEV), status_word()
    td, pd, one = table.to(DEV), pairs.to(DEV), torch.ones(2, device=DEV)
    for runs in STEPS:
        T = sum(n for _, n in runs)
        for rep in range(2 if max(n for _, n in runs) <= DEPTH else 1):                    # a repeated short step changes nothing
            x = torch.zeros(T, 2, W, device=DEV)
            ops.hyper_rows(x, W, T, f32=True, eps=1e-5, tokens=i32(sum((toks[s][p:p + n] for s, (p, n) in enumerate(runs)), [])), table=td,
                           pairs=(pd, spec["mul_prev"], spec["mul_cur"], recent), meta=meta(runs, slots), n_seq=3, next_in=one, status=st)
        w = torch.cat([want[s][p:p + n] for s, (p, n) in enumerate(runs)])
        assert torch.equal(x[:, 0].cpu(), w) and torch.equal(x[:, 1].cpu(), w) and int(st[0]) == 0, runs


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dim,vdim,taps,rot,inter,norm,own_v,bias", [
    (3, 1, 40, 24, 0, 12, True, "", True, True), (6, 2, 48, 48, 3, 32, True, "whole", False, False), (4, 2, 128, 128, 4, 128, False, "", True, True),
    (7, 7, 33, 45, 5, 22, False, "", True, True), (20, 3, 96, 96, 2, 64, False, "whole", True, True), (2, 1, 256, 200, 1, 64, False, "head", True, False),
    (5, 5, 27, 27, 6, 2, True, "whole", False, False), (1, 1, 250, 250, 2, 250, True, "whole", False, True), (2, 2, 14, 3, 0, 0, False, "", True, False)])
def test_conv_norm_rotation_across_portions(H, G, dim, vdim, taps, rot, inter, norm, own_v, bias, f32):
    """Bias, convolution, norms of both kinds, both layouts of the rotation, values of their own or the keys: every portion equals the whole sequence."""
    torch.manual_seed(2)
    dt, tol, eps = (torch.float32, 4e-6, 1e-3) if f32 else (torch.bfloat16, 6e-3, 1e-3)
    up = lambda n: -(-n // 64) * 64
    dp, dvp, C = up(dim), up(vdim), (H + G) * dim + (G * vdim if own_v else 0)
    slots, L, base = [2, 0, 3], 240, 300.0
    u = [torch.randn(L, C).to(dt).float() for _ in slots]
    w, b = torch.randn(C, taps) if taps else None, torch.randn(C) if bias else None
    gq, gk = torch.randn(H * dim if norm == "whole" else dim), torch.randn(G * dim if norm == "whole" else dim)
    want = []
    for x in u:
        y = x + b if bias else x
        y = causal_conv(y, w) if taps else y
        q, k = y[:, :H * dim], y[:, H * dim:(H + G) * dim]
        v = (y[:, (H + G) * dim:] if own_v else k).reshape(L, G, vdim)
        if norm == "whole":
            q, k = rms_norm(q, gq, eps), rms_norm(k, gk, eps)
        q, k = q.reshape(L, H, dim), k.reshape(L, G, dim)
        if norm == "head":
            q, k = rms_norm(q, gq, eps), rms_norm(k, gk, eps)
        want.append((oracle.rotate(q, rot, base, inter), oracle.rotate(k, rot, base, inter), v))
    ring = torch.full((4, taps - 1 + DEPTH, C), 50.0, dtype=dt, device=DEV) if taps else None            # what another sequence left behind
    cache, st = torch.full((700, G * (dp + dvp) + 64), 9.0, dtype=dt, device=DEV), status_word()
    dev = lambda t: t.to(DEV).contiguous() if t is not None else None
    for runs in STEPS:
        T = sum(n for _, n in runs)
        where = torch.randperm(700, generator=torch.Generator().manual_seed(T))[:T].tolist()
        proj = torch.full((T, -(-C // 8) * 8 + 16), 77.0, dtype=dt, device=DEV)
        proj[:, :C] = torch.cat([u[s][p:p + n] for s, (p, n) in enumerate(runs)]).to(dt)
        pos = [p + i for p, n in runs for i in range(n)]
        ang = torch.tensor(pos, dtype=torch.float64)[:, None] * torch.tensor([base ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64)
        table = torch.stack([ang.cos(), ang.sin()], -1).float().to(DEV) if rot else None
        q = torch.zeros(T, H * dp, dtype=dt, device=DEV)
        for rep in range(2 if max(n for _, n in runs) <= DEPTH else 1):
            ops.conv_qkv(proj, dev(w.T) if taps else None, dev(gq), dev(gk), table, ring, q, cache, meta(runs, slots, where), H=H, G=G, dim=dim, dp=dp, vdim=vdim, dvp=dvp,
                         pairs=rot // 2, eps=eps, n_seq=3, max_q_len=max(n for _, n in runs), bias=dev(b), norm=norm, half=not inter, values_are_keys=not own_v, n_slots=4, status=st)
        assert int(st[0]) == 0
        row = 0
        for s, (p, n) in enumerate(runs):
            got = q[row:row + n].view(n, H, dp)
            assert rel(got[..., :dim], want[s][0][p:p + n]) < tol and float(got[..., dim:].abs().sum()) == 0, runs
            c = cache[torch.tensor(where[row:row + n], device=DEV)]
            assert rel(c[:, :G * dp].view(n, G, dp)[..., :dim], want[s][1][p:p + n]) < tol, runs
            assert rel(c[:, G * dp:G * (dp + dvp)].view(n, G, dvp)[..., :vdim], want[s][2][p:p + n]) < tol, runs
            assert float((c[:, G * (dp + dvp):] - 9).abs().sum()) == 0
            row += n


@pytest.mark.parametrize("H,G,dim,vdim,window,keep,splits,sink,gate", [
    (8, 1, 128, 72, 90, 20, 2, True, ""), (3, 3, 40, 24, 1, 1, 1, True, "head"), (6, 2, 64, 64, 64, 64, 3, False, "value"), (9, 1, 200, 256, 65, 130, 4, True, "value"),
    (5, 1, 192, 33, 63, 5, 1, False, "head"), (40, 1, 100, 192, 130, 3, 5, True, ""), (12, 4, 256, 128, 0, 0, 5, True, "value"), (128, 1, 16, 48, 100, 65, 6, False, "head"),
    (4, 2, 130, 136, 4096, 7, 7, True, "value"), (6, 3, 96, 96, 50, 700, 3, False, "head"), (2, 1, 64, 64, 70, 129, 2, True, "")])
def test_attention_with_kept_keys_sinks_and_gates(H, G, dim, vdim, window, keep, splits, sink, gate):
    """Ragged batch on scattered pages; rows point at the first key of their window, at the one just in front of it, at the last kept key and the next
    one - the tcgen05 kernels and the ordinary-core one.  Where no visible key stands out, the sink takes most of the weight."""
    torch.manual_seed(5)
    lens, q_lens = [333, 64, 193, 1, 65], [130, 1, 2, 1, 65]
    dt, scale, factor = torch.bfloat16, 0.7, 1.3
    pg = Paged(lens, G, dim, vdim, dt)
    T, group = sum(q_lens), H // G
    starts = [sum(q_lens[:i]) for i in range(len(q_lens))]
    q = torch.zeros(T, H, pg.dp)
    q[..., :dim] = torch.randn(T, H, dim) * 0.1
    for s, (n, m) in enumerate(zip(lens, q_lens)):
        for i in range(m):
            pos, w = n - m + i, window or n
            keys = [k for k in (pos - w + 1, pos - w, keep - 1, keep, pos - w + 2, pos - w - 1, 0, 63, 64, pos, pos - 1, keep + 1) if 0 <= k <= pos]
            for h in range(H):
                if (i + h) % 5:
                    k = pg.k[s][keys[(i * 3 + h) % len(keys)], h // group]
                    q[starts[s] + i, h, :dim] += k * (14.0 / float(k @ k))
    q = q.to(dt)
    qd, ldo, st = q.reshape(T, -1).to(DEV), -(-(H * vdim) // 8) * 8, status_word()
    snk = torch.randn(H) * 2 + 3.0 if sink else None
    gw = {"": 0, "head": H, "value": H * vdim}[gate]
    g = torch.randn(T, gw + 3).to(dt)
    gd, sd = g.to(DEV), snk.to(DEV) if sink else None
    extras = ops.attn_extras(sink=sd, gate=gd[:, 2:] if gate else None, per_value=gate == "value", keep_first=keep, out_scale=factor)      # not on 16 bytes
    kw = dict(T=T, n_seq=len(lens), Hq=H, Hkv=G, dp=pg.dp, dvp=pg.dvp, dv=vdim, window=window, scale=scale, extras=extras, status=st)
    where = (pg.table, i32(lens), i32(starts), i32(q_lens))
    maps = ops.encode_window_maps(pg.store, G, pg.dp, pg.dvp)
    new = lambda: torch.full((T, ldo), 7.0, dtype=dt, device=DEV)
    outs = {"simt": new()}
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
        see = oracle.visible(n, window or None, keep)
        want = oracle.attend(full, pg.k[s], pg.v[s], scale, see, snk)[n - m:] * factor
        ref = want.norm(dim=-1)
        if sink:
            ref = ref + 0.2 * oracle.attend(full, pg.k[s], pg.v[s], scale, see, None)[n - m:].norm(dim=-1) * factor       # what is left beside a strong sink
        if gate:
            gs = torch.sigmoid(g[starts[s]:starts[s] + m, 2:2 + gw].float())
            want, ref = (want * gs[:, :, None], ref * gs) if gate == "head" else (want * gs.view(m, H, vdim), ref * gs.view(m, H, vdim).pow(2).mean(-1).sqrt())
        for name, o in outs.items():
            o = o[starts[s]:starts[s] + m].float().cpu()
            err = (o[:, :H * vdim].reshape(m, H, vdim) - want).norm(dim=-1) / ref
            assert float(err.max()) < 3e-2, (name, s, float(err.max()))
            assert float((o[:, H * vdim:] - 7).abs().sum()) == 0


def scan_buffers(H, d, dv, n_state=4):
    vp = -(-dv // 4) * 4
    g = torch.Generator(device=DEV).manual_seed(3)
    state = torch.empty(n_state, 2, H, d, vp, device=DEV).normal_(0, 30, generator=g)
    tags = torch.randint(-1, 300, (n_state, H, 2), dtype=torch.int32, device=DEV, generator=g)
    return state, tags, torch.empty(n_state, DEPTH, H, 2 * d + vp, device=DEV).normal_(0, 30, generator=g)


SHORT, CHUNKS, FP32 = "short", "chunks", "fp32"
LONG_STEPS = [[(0, 400), (0, 2), (0, 17)], [(400, 3), (2, 300), (17, 128)], [(403, 256), (302, 1), (145, 129)], [(659, 1), (303, 270), (274, 8)], [(660, 33), (573, 130), (276, 385)]]


@pytest.mark.parametrize("form", [FP32, SHORT, CHUNKS])
@pytest.mark.parametrize("kind,H,d,dv,rot,tau,rank,harsh", [
    ("retention", 3, 24, 40, 16, 0, 0, True), ("retention", 1, 13, 7, 6, 0, 0, False), ("retention", 2, 128, 256, 128, 0, 0, True), ("retention", 6, 32, 64, 0, 0, 0, True),
    ("retention", 2, 72, 200, 20, 0, 0, False), ("gla", 4, 20, 36, 0, 8.0, 5, False), ("gla", 3, 9, 17, 0, 1.0, 1, True), ("gla", 2, 256, 64, 0, 16.0, 16, True),
    ("gla", 2, 64, 128, 0, 2.0, 33, False), ("gla", 2, 128, 256, 0, 16.0, 16, False), ("gla", 2, 96, 64, 0, 4.0, 8, True)])
def test_linear_attention_across_portions(kind, H, d, dv, rot, tau, rank, harsh, form):
    """Rotation, decays, recurrence, output norm and gate of every portion equal those of the whole sequence, wherever it is cut and after steps back;
    heads that remember for hundreds of tokens, with `harsh` beside channels that forget at once."""
    torch.manual_seed(6)
    f32 = form == FP32
    dt, tol, eps, base, factor = torch.float32 if f32 else torch.bfloat16, 1e-5 if f32 else 8e-3, 1e-3, 200.0, 1.7
    slots, L = [1, 3, 0], 704
    rd = lambda *s: torch.randn(*s).to(dt).float()
    up = lambda n: -(-n // 8) * 8
    decay = torch.tensor([([0.999, 0.0, 0.97, 0.25, 1.0, 0.9] if harsh else [0.9990234375, 0.5])[h % (6 if harsh else 2)] for h in range(H)])
    a2, a2b = torch.randn(H * d, max(rank, 1)) * max(rank, 1) ** -0.5, torch.randn(H * d) * 2 + (2 if harsh else 4)
    a2[0], a2b[0] = 0, 30.0                                        # a channel that forgets nothing
    if harsh:
        a2[H * d - 1], a2b[H * d - 1] = 0, -60.0                   # and one that forgets at once
    norm = torch.randn(dv) + 1 if kind == "gla" else None
    widths = {"q": H * d, "k": H * d, "v": H * dv, "g": H * dv, "a1": rank}
    at, cols = 8, {}
    for n, w in widths.items():
        cols[n], at = at, at + up(w)
    seqs, want = [], []
    for _ in slots:
        x = {n: rd(L, w) for n, w in widths.items() if w}
        q, k, v = x["q"].double().view(L, H, d), x["k"].double().view(L, H, d), x["v"].double().view(L, H, dv)
        if kind == "retention":
            q, k, al = oracle.rotate(q, rot, base, False), oracle.rotate(k, rot, base, False) * d ** -0.5, decay.double()[None, :, None].expand(L, H, d)
        else:
            z = x["a1"].double() @ a2.double().T + a2b.double()
            q, al = q * d ** -0.5, torch.sigmoid(z).pow(1 / tau).view(L, H, d)
        o = oracle.linear_attention(q, k, v, al)
        o = rms_norm(o, norm.double() if norm is not None else torch.ones(dv).double(), eps).reshape(L, -1) * oracle.silu(x["g"].double()) * factor
        seqs.append(x)
        want.append(o.float())
    dev = lambda t: t.float().to(DEV).contiguous() if t is not None else None
    dec, a2d, a2bd, nd = dev(decay), dev(a2), dev(a2b), dev(norm)
    state, tags, ring = scan_buffers(H, d, dv)
    st = status_word()
    scratch = ops.scan_scratch(600, 3, H, d, dv, DEV) if form == CHUNKS else None
    if scratch:
        scratch[0].fill_(float("nan")); scratch[1].fill_(float("nan"))
    back = [[(194, 8), (79, 8), (221, 8)], [(195, 30), (86, 9), (222, 1)]]                   # long runs behind rejected rows
    for runs in STEPS + back + [[(0, 1), (0, 17), (0, 400)]] + [r for r in LONG_STEPS]:
        T = sum(n for _, n in runs)
        proj = torch.full((T, at), 77.0, dtype=dt, device=DEV)
        for n, w in ((n, w) for n, w in widths.items() if w):
            proj[:, cols[n]:cols[n] + w] = torch.cat([seqs[s][n][p:p + m] for s, (p, m) in enumerate(runs)]).to(dt)
        pos = [p + i for p, n in runs for i in range(n)]
        ang = torch.tensor(pos, dtype=torch.float64)[:, None] * torch.tensor([base ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64)
        table = torch.stack([ang.cos(), ang.sin()], -1).float().to(DEV) if rot else None
        out = torch.full((T, up(H * dv) + 8), 5.0, dtype=dt, device=DEV)
        for rep in range(2 if max(n for _, n in runs) <= DEPTH else 1):
            arg = ops.decay_scan_arg(*(proj[:, cols[n]:] for n in ("q", "k", "v", "g")), state, tags, ring, out, meta(runs, slots), H=H, dim=d, vdim=dv, n_seq=3,
                                     max_q_len=max(n for _, n in runs), eps=eps, rope=table, pairs=rot // 2, q_scale=d ** -0.5 if kind == "gla" else 1.0,
                                     k_scale=1.0 if kind == "gla" else d ** -0.5, decay=dec if kind == "retention" else None,
                                     low_rank=(proj[:, cols["a1"]:], a2d, a2bd) if kind == "gla" else None, tau=tau or 1.0, norm=nd, out_scale=factor, chunks=scratch, T=T, status=st)
            ops.decay_scan(arg, f32=f32)
        assert int(st[0]) == 0, runs
        row = 0
        for s, (p, n) in enumerate(runs):
            e = (out[row:row + n, :H * dv].float().cpu() - want[s][p:p + n]).view(n, H, dv).norm(dim=-1) / want[s].view(L, H, dv).norm(dim=-1).mean(0)
            assert float(e.max()) < 3 * tol, (runs, s, float(e.max()))
            row += n
        assert float((out[:, H * dv:] - 5).abs().sum()) == 0


def test_a_state_at_another_position_is_reported():
    H, d, dv = 1, 8, 8
    state, tags, ring = scan_buffers(H, d, dv)
    tags.fill_(40)
    proj, out, st = torch.zeros(1, 64, device=DEV), torch.zeros(1, 8, device=DEV), status_word()
    col = lambda i: proj[:, 8 * i:]
    arg = ops.decay_scan_arg(col(0), col(1), col(2), col(3), state, tags, ring, out, meta([(30, 1)], [2]), H=H, dim=d, vdim=dv, n_seq=1, max_q_len=1, eps=1e-5,
                             decay=torch.ones(1, device=DEV), status=st)
    ops.decay_scan(arg, f32=True)
    assert int(st[0]) >> 24 == 5


@pytest.mark.parametrize("T", [3, 40, 200])
@pytest.mark.parametrize("E,k,groups", [(12, 3, (4, 2)), (8, 3, (8, 5)), (16, 4, None), (9, 9, (3, 3))])
def test_routing_with_unnormalised_sigmoid_weights(T, E, k, groups):
    torch.manual_seed(7)
    logits = torch.randn(T, E)
    idx, wts = torch.zeros(T, k, dtype=torch.int32, device=DEV), torch.zeros(T, k, device=DEV)
    n, keep = groups or (1, 1)
    ops.router_select(logits.to(DEV), None, idx, wts, T, k, "sigmoid", False, 1.0, n, keep)
    for t in range(T):
        s = torch.sigmoid(logits[t])
        want = oracle.choose_experts(s, k, {"count": n, "keep": keep})
        assert sorted(idx[t].tolist()) == sorted(want) and torch.allclose(wts[t].cpu(), s[idx[t].long().cpu()], atol=1e-6)


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_silu_rows(dt):
    g, u = torch.randn(5, 1037).to(dt), torch.randn(5, 1037).to(dt)
    out = torch.zeros(5, 1037, dtype=dt, device=DEV)
    ops.silu_rows(g.to(DEV), u.to(DEV), out, 5)
    assert rel(out, oracle.silu(g.float()) * u.float()) < (1e-6 if dt == torch.float32 else 4e-3)


# ------------------------------------------------------------------ engine
def logits(cfg, t, toks):
    return oracle.logits(cfg, {k: v.double() for k, v in t.items()}, toks).float()


def build(cfg, tmp_path, dtype="float32", seed=0, max_tokens=2048, live=4, tensors=None, rank=6):
    from cuteafd_b200.serving.trace import TraceReplay
    t = tensors or make_tensors(cfg, seed, rank)
    p = write_snapshot(cfg, t, tmp_path / f"{dtype}{seed}")
    rep = TraceReplay(str(p), dtype=dtype, max_tokens=max_tokens, max_live=live)
    g = torch.Generator(device=DEV).manual_seed(9)      # what earlier owners of a page or a state slot could have left behind: large, finite
    for buf in [rep.engine.kv] + rep.engine.state_buffers():
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
    else:      # (the norm behind a linear mixer divides by a product of two rows: where that is nearly zero, rounding turns its sign)
        assert int((e > 0.2).sum()) <= max(1, len(e) // 100) and float(e.median()) < 0.04, (float(e.max()), float(e.median()), int((e > 0.2).sum()))


def steady(cfg, dtype):
    """For bf16 runs: every expert is chosen (as many per token as there are), so that rounding turns no close decision; their weights still differ."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if dtype == "bfloat16" and (layer["mlp"] or {}).get("kind") == "moe":
            r = layer["mlp"]["router"]
            r["top"] = r["experts"]
            if r.get("groups"):
                r["groups"]["keep"] = r["groups"]["count"]
    return cfg


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompts_portions_and_decoding_match_the_oracle(name, dtype, tmp_path):
    cfg = steady(CONFIGS[name], dtype)
    rep, t = build(cfg, tmp_path, dtype, rank=RANK[name])
    toks = tokens(cfg, 230, 1)
    want = logits(cfg, t, toks)
    rep.engine.tap = [] if dtype == "float32" else None
    whole = run_portions(rep, "a", toks, [len(toks)])
    check(whole, want, dtype)
    if dtype == "float32":
        taps, ref = rep.engine.tap, [x.float() for x in oracle.hidden_states(cfg, {k: v.double() for k, v in t.items()}, toks)]
        assert len(taps) == len(ref) and all(rel(a, b) < 1e-5 for a, b in zip(taps, ref))
        rep.engine.tap = None
    for i, cuts in enumerate(([160, 1], [2, 2, 3, 57, 64, 2, 63, 2, 9, 8, 7, 1, 65], [1], [64, 64, 1], [33], [130, 98, 2])):
        check(run_portions(rep, f"p{i}", toks, cuts), want, dtype)
    assert rep.pool.n_free == rep.pool.n_pages - 1 and len(rep.runner._free_slots) == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_of_unequal_requests_equal_each_alone_and_pages_and_slots_are_reused(dtype, tmp_path):
    cfg = steady(MIXED, dtype)
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


WINDOW, KEEP = 100, 70


def pointing(kind):
    """One layer whose second head, at rows of token 6, looks for token 5: two channels that only these tokens have decide its scores, behind a rotation
    that leaves the last dimension alone.  Every other token's rows are the same to it."""
    a = attn(2, 1, 40, 40, 0.3, 12, window=WINDOW, keep=KEEP, conv=3 if kind == "parallel_2" else None)
    layer = {"parallel": parallel(a, retention(1, 8, 8, 0), (1.0, 0.1), None), "parallel_2": parallel2(a, gla(1, 8, 8, 4.0), None),
             "attention": plain({k: v for k, v in dict(a, conv=2).items() if k != "mask"}, None)}[kind]
    cfg = variant(PLAIN, layers=[layer], width=96, vocab=61, streams=2)
    t = make_tensors(cfg, 7)
    p = "l0.mix" if kind == "attention" else "l0.mix.left"
    t["embed"][5] = torch.roll(t["embed"][7], 11)
    t["embed"][:, :2] = 0
    t["embed"][5, 0], t["embed"][6, 1] = 4.0, 4.0
    t["l0.norm1"][:2] = 1.0
    for k, row, ch in (("q", 40 + 39, 1), ("k", 39, 0)):
        t[f"{p}.{k}"][:, :2] = 0
        t[f"{p}.{k}"][row] = 0
        t[f"{p}.{k}"][row, ch] = 3.0 if kind != "parallel_2" else 60.0
        if f"{p}.{k}.b" in t:
            t[f"{p}.{k}.b"][row] = 0
        if f"{p}.{k}.conv" in t:
            t[f"{p}.{k}.conv"][row] = 0
            t[f"{p}.{k}.conv"][row, -1] = 1.0
        if f"{p}.{k}.norm" in t:
            t[f"{p}.{k}.norm"][row] = 2.0
    if f"{p}.sink" in t:
        t[f"{p}.sink"][:] = -1.0
    return cfg, {k: v.to(torch.bfloat16).float() for k, v in t.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["parallel", "parallel_2", "attention"])
def test_one_key_decides_inside_the_window_and_among_the_kept_ones(kind, dtype, tmp_path):
    """One score stands out: a key just inside the window or the last kept one must count, one just outside or the next must not - in prompts, portions
    and decoding, next to page borders too."""
    cfg, t = pointing(kind)
    rep, t = build(cfg, tmp_path, dtype, tensors=t)
    n = 300
    base = [x if x not in (5, 6) else 7 for x in tokens(cfg, n, 8)]
    seen = {True: 0, False: 0}
    for q in (WINDOW + KEEP - 1, WINDOW + KEEP, 191, 192, 255, 256, 298):
        base_q = list(base)
        base_q[q] = 6
        alone = logits(cfg, t, base_q)
        for k in (q - WINDOW + 1, q - WINDOW, KEEP - 1, KEEP, 0, q - 1, KEEP + 1):
            if not 0 <= k < q:
                continue
            toks = list(base_q)
            toks[k] = 5
            want = logits(cfg, t, toks)
            moved, inside = float(errors(alone[q:q + 1], want[q:q + 1])), kind == "attention" or q - k < WINDOW or k < KEEP
            assert moved > 0.15 if inside else moved < 0.1, (q, k, moved)
            seen[inside] += 1
            for cuts in ([n], [q, 1, 2]) if k in (q - WINDOW, q - WINDOW + 1, KEEP, KEEP - 1) else ([q - 1, 2],):
                got = run_portions(rep, "x", toks, cuts)
                e = float(errors(got[q:q + 1], want[q:q + 1]))
                assert e < (1e-4 if dtype == "float32" else 0.04), (q, k, cuts, e)
    assert seen[True] > 10 and (kind == "attention" or seen[False] > 5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["retention", "gla"])
def test_the_first_token_is_remembered_for_hundreds_of_tokens(kind, dtype, tmp_path):
    """A linear mixer that forgets nothing: the first token still shows at the end, through whole prompts, portions and decoding; a state that is lost
    or taken from another slot would too."""
    a = attn(1, 1, 16, 16, 0.3, 0, window=1)
    layer = parallel(a, retention(2, 16, 16, 0, decay=[1.0, 1.0]), (0.1, 1.5), None) if kind == "retention" else parallel2(dict(a, conv=2), gla(2, 16, 16, 16.0), None)
    cfg = variant(PLAIN, layers=[layer], width=64, vocab=61, streams=2)
    t = make_tensors(cfg, 17)
    if kind == "gla":
        t["l0.mix.right.a2"][:], t["l0.mix.right.a2.b"][:] = 0, 40.0
    # the value of token 5 is a direction of its own, far larger than the others', and every key and query agree in one channel
    t["embed"][:, :2], t["embed"][:, 1] = 0, 2.0
    t["embed"][5, 0] = 6.0
    t["l0.norm1"][:2] = 1.0
    for k in ("q", "k"):
        t[f"l0.mix.right.{k}"] *= 0.2
        t[f"l0.mix.right.{k}"][:, 1] = 1.0
    t["l0.mix.right.v"] *= 0.1
    t["l0.mix.right.v"][:, 0] = torch.randn(32, generator=torch.Generator().manual_seed(3)) * 6.0
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
        rep, t = build(CONFIGS[name], tmp_path / name, "float32", rank=RANK[name])
        for n in (1, 2, 3):
            toks = tokens(CONFIGS[name], n, 20 + n)
            check(run_portions(rep, f"r{n}", toks, [n]), logits(CONFIGS[name], t, toks), "float32")


@pytest.mark.parametrize("name", ["wide", "mixed"])
def test_long_decoding_crosses_pages_windows_and_split_counts(name, tmp_path):
    cfg = steady(CONFIGS[name], "bfloat16")
    rep, t = build(cfg, tmp_path, "bfloat16", rank=RANK[name])
    toks = tokens(cfg, 300, 30)
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
    pos = 0
    for keep, drafted in ((2, 8), (66, 66), (3, 8), (1, 2), (7, 8), (8, 8), (1, 8), (1, 8), (1, 8), (2, 5), (4, 7), (1, 1), (5, 8)):
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
    cfg = MIXED
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


def test_random_weights_of_a_named_shape_run(tmp_path):
    """The synthetic preset at a small size: prefill and decode through the generator, bf16."""
    from cuteafd_b200.config import vozetar_spec
    from cuteafd_b200.engine.generate import generate
    from cuteafd_b200.engine.registry import build_engine
    from cuteafd_b200.models.hyper_stack import hyper_weights_random
    spec = vozetar_spec(n_layers=4, hidden=256, heads=4, kv_heads=2, ff=512, window=128, rec_heads=2, rec_dim=64, rec_vdim=128, experts=16, expert_ff=128, streams=3)
    eng = build_engine(spec, hyper_weights_random(spec, torch.device(DEV)), n_pages=24, max_seqs=2, max_pages_per_seq=8)
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

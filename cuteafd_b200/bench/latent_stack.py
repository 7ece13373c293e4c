"""Prefill and decode of a latent-attention stack (the Bedovik design) beside the closest other model of the framework at equal size: the
multi-head latent attention stack with a rotated part and gated experts (`engine.mla`), same widths, heads, latent, experts per token,
layer runs and weights per expert.  bf16 weights on both sides, random, one GPU.

    python bench.py --config bedovik                                   # every size, both models, one JSON line
    python bench.py --config bedovik --bedovik-size medium
    python -m cuteafd_b200.bench.latent_stack --size medium --kernels  # plus device time and share of the roofline per launch site

Throughput: CUDA events on the launching stream around `steps` graph replays (decode) or eager chunks (prefill) after warm-up; weights
are far larger than L2.  Per-launch times (`--kernels`): every entry point of the native library is bracketed by events while one eager
step is enqueued behind a delay, so the GPU runs the launches back to back; the roofline of a launch is the slower of its operations
over the measured bf16 peak and its bytes over the measured copy bandwidth (`MEASURED_PEAKS.json`).
"""
from __future__ import annotations

import argparse
import collections
import dataclasses
import gc
import json
import os

import torch

from ..config import AttentionSpec, ModelSpec, QuantSpec, bedovik_spec
from ..engine.engine import PAGE, StepShape
from ..engine.generate import BatchGenerator
from ..engine.kv import PagePool, SeqKV
from ..engine.registry import build_engine, load_weights
from ..ops import native

# hidden, heads, latent rank, experts, squared-ReLU width, layers (the middle half of them twice)
SIZES = {"small": (2048, 16, 512, 64, 1536, 8), "medium": (4096, 32, 512, 64, 1536, 4), "large": (7168, 128, 512, 32, 3072, 4)}


def specs(size: str) -> tuple[ModelSpec, ModelSpec]:
    hidden, heads, rank, experts, ff, layers = SIZES[size]
    ours = bedovik_spec(n_layers=layers, heads=heads, hidden=hidden, rank=rank, experts=experts, ff=ff)
    mla = ModelSpec(name="mla-equal", family="deepseek_v3", vocab=ours.vocab, hidden=hidden, n_layers=len(ours.layer_runs()), rms_eps=1e-6,
                    attn=AttentionSpec(kind="mla", n_heads=heads, n_kv_heads=heads, head_dim=192, kv_lora_rank=rank, qk_nope_head_dim=128, qk_rope_head_dim=64,
                                       v_head_dim=128),
                    moe=dataclasses.replace(ours.moe, activation="swiglu", group_score="top2", intermediate=ff * 2 // 3, first_dense=0),
                    quant=QuantSpec(experts="bf16", dense="bf16", kv="bf16"))
    return ours, mla


def make_engine(spec: ModelSpec, pages: int, seqs: int, per_seq: int):
    dev = torch.device("cuda", 0)
    if spec.attn.kind == "mla":
        from ..engine.mla import mla_weights_random
        w = mla_weights_random(spec, dev, distinct_moe_layers=4, seed=1)
    else:
        w = load_weights(spec.name, spec, dev)
    eng = build_engine(spec, w, n_pages=pages, max_seqs=seqs, max_pages_per_seq=per_seq)
    for t in eng.cache_buffers() if hasattr(eng, "cache_buffers") else [eng.kv]:
        t.normal_(0, 1)
    return eng


def timed(fn, n: int, warm: int) -> float:
    for _ in range(warm):
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(n):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / n


def decode_shape(eng, batch: int, context: int, pool: PagePool) -> tuple:
    gen = BatchGenerator(eng, pool)
    gen.seqs, gen.hist = [], None
    for _ in range(batch):
        s = SeqKV()
        s.ensure(pool, context + 2)
        s.length = context
        gen.seqs.append(s)
    gen.last = torch.randint(0, eng.spec.vocab, (batch,), generator=torch.Generator().manual_seed(0)).tolist()
    return gen, gen.plan_decode()


def prefill_shape(eng, chunk: int, context: int, pool: PagePool) -> tuple:
    s = SeqKV()
    s.ensure(pool, context)
    off = context - chunk
    toks = torch.randint(0, eng.spec.vocab, (chunk,), generator=torch.Generator().manual_seed(0)).tolist()
    eng.set_inputs(toks, list(range(off, context)), [s.slot(p) for p in range(off, context)], [chunk - 1], [context], [0], [chunk], [s.pages])
    return s, StepShape(T=chunk, n_seq=1, max_q_len=chunk, n_logits=1, attn_splits=1)


# ------------------------------------------------------------------ per-launch times
def launch_times(eng, sh, reps: int = 3) -> dict:
    """{site: [launches per step, milliseconds per step]} of eager steps; a site is an entry point plus the shape of its product."""
    lib, names = native.lib(), [n for n in native._PROTOS if hasattr(native.lib(), n) and "encode" not in n and "capacity" not in n]
    real = {n: getattr(lib, n) for n in names}
    log: list = []

    def site(n, a):
        if n == "cuteafd_tc_linear":
            return ("gemm", "grouped" if a[12] else "dense", "swiglu" if a[1] else "", a[19], a[20])
        return (n.replace("cuteafd_", ""),)

    def wrap(n):
        def run(*a):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            rc = real[n](*a)
            e1.record()
            log.append((site(n, a), e0, e1))
            return rc
        return run
    acc: dict = collections.defaultdict(lambda: [0, 0.0])
    try:
        for n in names:
            setattr(lib, n, wrap(n))
        for rep in range(reps + 1):
            log.clear()
            torch.cuda.synchronize()
            torch.cuda._sleep(60_000_000)                     # the step is enqueued behind this delay
            eng.run(sh, use_graph=False)
            torch.cuda.synchronize()
            if rep == 0:
                continue                                      # warm-up
            for key, e0, e1 in log:
                acc[key][0] += 1
                acc[key][1] += e0.elapsed_time(e1)
    finally:
        for n in names:
            setattr(lib, n, real[n])
    return {k: [c / reps, t / reps] for k, (c, t) in acc.items()}


def roofline(spec: ModelSpec, T: int, pairs: int, kv_rows: int, site: tuple, prefill: bool, peaks: dict) -> tuple | None:
    """(label, ideal milliseconds of one launch) by what a launch has to compute and move; None = control work without a bound."""
    a, m, W = spec.attn, spec.moe, spec.hidden
    H, r, k = a.n_heads, a.kv_lora_rank, m.top_k
    tf, bw = peaks["bf16_tflops"] * 1e9, peaks["hbm_gbs"] * 1e6            # per millisecond
    lo = lambda ops, nbytes: max(ops / tf, nbytes / bw)
    if site[0] == "gemm":
        _, form, sw, N, K = site
        if form == "grouped":
            if N == m.intermediate or K == m.intermediate:                 # experts
                act = min(m.n_experts, T * k) if T * k < 4 * m.n_experts else m.n_experts
                mats = 2 if sw else 1
                return ("experts up" if N == m.intermediate else "experts down", lo(2.0 * T * k * N * K * mats, 2.0 * (act * N * K * mats + T * k * (N + K))))
            return ("q -> latent" if N >= r else "latent -> v", lo(2.0 * T * H * N * K, 2.0 * (H * N * K + T * H * (N + K))))
        if N == spec.vocab:
            return ("head", lo(2.0 * N * K, 2.0 * N * K))
        if K == 2 * W:
            return ("loop entry", lo(2.0 * T * N * K, 2.0 * N * K + T * (2.0 * K + 4.0 * N)))
        if K == r and N > W:
            return ("context -> keys, values", lo(2.0 * kv_rows * N * K, 2.0 * (N * K + kv_rows * (N + K))))
        if N == W:
            return ("output projection", lo(2.0 * T * N * K, 2.0 * (N * K + T * (N + K))))
        return ("input projections", lo(2.0 * T * N * K, 2.0 * N * K + T * (2.0 * K + 4.0 * N)))
    n = site[0]
    dq, dv = (128 + (64 if a.kind == "mla" else 0)), 128
    row = r + (64 if a.kind == "mla" else 0)
    if n in ("latent_attention", "mla_attention"):
        return ("attention (absorbed)", lo(2.0 * pairs * H * (row + r), 2.0 * (kv_rows * row + T * H * (row + r))))
    if n in ("latent_prefill_attention", "mla_prefill_attention"):
        return ("attention (expanded)", lo(2.0 * pairs * H * (dq + dv), 2.0 * (kv_rows * H * 256 + T * H * (dq + dv))))
    if n in ("latent_gather_ctx", "mla_gather_ctx"):
        return ("context gather", lo(0, 4.0 * kv_rows * row))
    if n in ("stack_combine", "moe_combine", "moe_combine_norm"):
        return ("combine (+ next norm)", lo(0, T * W * ((2 + 2.0 * k + 8 + 2) if n == "stack_combine" else (2.0 * k + 4 + 2))))
    if n in ("latent_prepare",):
        width = H * 128 + r + H + m.n_experts
        return ("projection split", lo(0, T * (4.0 * width + 2.0 * (H * 128 + r) + 4.0 * m.n_experts)))
    if n in ("mla_q_split", "mla_kv_prepare"):
        return ("projection split", lo(0, T * 4.0 * (H * 192 if n == "mla_q_split" else row)))
    if n in ("add_rmsnorm",):
        return ("norm", lo(0, 4.0 * T * W))
    if n == "head_to_token_major":
        return ("head-major -> token-major", lo(0, 4.0 * T * H * 128))
    if n == "gather_rows":
        return ("expert gather", lo(0, 4.0 * T * k * W))
    if n in ("stack_embed", "stack_stream"):
        return ("embedding / pass entry", lo(0, T * W * 10.0))
    if n == "router_logits":
        return ("router logits", lo(0, 2.0 * m.n_experts * W + 2.0 * T * W))
    return None


def kernel_table(eng, sh, pairs: int, kv_rows: int, prefill: bool, peaks: dict, roofline=roofline) -> dict:
    out: dict = {}
    for s, (count, ms) in launch_times(eng, sh).items():
        r = roofline(eng.spec, sh.T, pairs, kv_rows, s, prefill, peaks)
        label, ideal = r if r else ("routing" if s[0].startswith("rout") else s[0], None)
        o = out.setdefault(label, {"launches": 0.0, "ms": 0.0, "ideal_ms": 0.0})
        o["launches"] += count
        o["ms"] += ms
        o["ideal_ms"] = None if ideal is None or o["ideal_ms"] is None else o["ideal_ms"] + ideal * count
    return {k: {"launches": round(v["launches"], 1), "us_per_launch": round(1e3 * v["ms"] / v["launches"], 1), "ms": round(v["ms"], 3),
                "roofline": round(v["ideal_ms"] / v["ms"], 3) if v["ideal_ms"] else None} for k, v in sorted(out.items(), key=lambda kv: -kv[1]["ms"])}


# ------------------------------------------------------------------ workloads
def measure(spec: ModelSpec, *, batches, context: int, chunks, steps: int, warmup: int, kernels: bool, peaks: dict, roofline=roofline, at_position=lambda eng, pos: None) -> dict:
    """`roofline`: what a launch has to compute and move, for the per-launch table (windowed layers see the last `attn.window` keys only).
    `at_position(engine, position)`: puts recurrent states that know their position in front of the step's first one."""
    win = spec.attn.window or 1 << 40
    seen = lambda lo, hi: sum(min(p + 1, win) for p in range(lo, hi))            # (query, key) pairs of positions [lo, hi)
    longest = max([context] + [c for _, c in chunks])
    per = longest // PAGE + 3
    pages = max(max(batches) * (context // PAGE + 2), per) + 2
    eng = make_engine(spec, pages, max(batches), per)
    res: dict = {"layer_runs": len(spec.layer_runs()), "weights_gb": round(eng.weights.nbytes() / 1e9, 2), "decode": [], "prefill": []}
    launches = 0
    for b in batches:
        pool = PagePool(pages)
        gen, sh = decode_shape(eng, b, context, pool)
        at_position(eng, context)
        ms = timed(lambda: eng.run(sh), steps, warmup)
        launches += eng.launches_per_step * steps
        row = {"batch": b, "context": context, "ms_per_step": round(ms, 4), "tokens_per_s": round(b / ms * 1e3, 1), "us_per_layer_run": round(1e3 * ms / res["layer_runs"], 1),
               "launches_per_step": eng.launches_per_step}
        if kernels:
            row["kernels"] = kernel_table(eng, sh, b * seen(context, context + 1), b * min(context + 1, win), False, peaks, roofline)
        res["decode"].append(row)
        eng.check_status()
    for chunk, ctx in chunks:
        s, sh = prefill_shape(eng, chunk, ctx, PagePool(pages))
        at_position(eng, ctx - chunk)
        ms = timed(lambda: eng.run(sh, use_graph=False), max(3, steps // 4), warmup)
        launches += eng.launches_per_step * max(3, steps // 4)
        row = {"chunk": chunk, "context": ctx, "ms_per_chunk": round(ms, 3), "tokens_per_s": round(chunk / ms * 1e3, 1), "us_per_layer_run": round(1e3 * ms / res["layer_runs"], 1)}
        if kernels:
            off = ctx - chunk
            row["kernels"] = kernel_table(eng, sh, seen(off, ctx), min(ctx, chunk + win), True, peaks, roofline)
        res["prefill"].append(row)
        eng.check_status()
    res["gpu_launches"] = launches
    return res


def peaks_used() -> dict:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    p = json.load(open(path)) if os.path.exists(path) else {}
    return {"bf16_tflops": float(p.get("bf16_tflops", 1590.0)), "hbm_gbs": float(p.get("hbm_gbs", 6650.0)), "source": "measured" if p else "fallback"}


def run(sizes=("small", "medium", "large"), *, batches=(16, 64), context: int = 4096, chunks=((4096, 4096), (2048, 16384)), steps: int = 20, warmup: int = 3,
        kernels: bool = False, clocks=None, only: str = "") -> dict:
    peaks = peaks_used()
    out = {"bench": "bedovik", "peaks": peaks, "sizes": {}}
    if clocks is not None:
        clocks.start()
    for size in sizes:
        hidden, heads, rank, experts, ff, layers = SIZES[size]
        entry = {"shape": {"hidden": hidden, "heads": heads, "latent": rank, "experts": experts, "top": 8, "expert_width": ff, "layers": layers}}
        for name, spec in zip(("bedovik", "mla"), specs(size)):
            if only and name != only:
                continue
            entry[name] = measure(spec, batches=batches, context=context, chunks=chunks, steps=steps, warmup=warmup, kernels=kernels, peaks=peaks)
            gc.collect()
            torch.cuda.empty_cache()
        out["sizes"][size] = entry
    if clocks is not None:
        out["clocks"] = clocks.stop()
    return out


def bench_line(args, clocks) -> dict:
    """The `bench.py --config bedovik` line: decode throughput of the largest measured size, everything else under `results`."""
    sizes = tuple(SIZES) if args.bedovik_size == "all" else (args.bedovik_size,)
    res = run(sizes, steps=args.steps, warmup=args.warmup, clocks=clocks)
    size = sizes[-1]
    d = res["sizes"][size]["bedovik"]["decode"][-1]
    ours, _ = specs(size)
    return {"metric": "decode_tokens_per_s", "value": d["tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
            "ms_per_step": d["ms_per_step"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16 operands, fp32 residual",
            "data": "synthetic token ids, random-init weights, context latents random-filled",
            "config": {"model": f"{ours.name} ({size})", "global_batch": d["batch"], "seq_len": d["context"], "parallelism": "single",
                       "l2": "weights far larger than L2; no flush needed"},
            "clocks": res.pop("clocks", None), "gpu_launches": sum(s["bedovik"]["gpu_launches"] for s in res["sizes"].values()), "results": res}


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--size", default="all", choices=["all", *SIZES])
    ap.add_argument("--steps", type=int, default=20); ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--context", type=int, default=4096); ap.add_argument("--batches", default="16,64")
    ap.add_argument("--chunks", default="4096:4096,2048:16384", help="prefill chunk:context pairs")
    ap.add_argument("--kernels", action="store_true"); ap.add_argument("--only", default="", choices=["", "bedovik", "mla"])
    a = ap.parse_args()
    chunks = tuple(tuple(int(x) for x in c.split(":")) for c in a.chunks.split(",") if c)
    print(json.dumps(run(tuple(SIZES) if a.size == "all" else (a.size,), batches=tuple(int(b) for b in a.batches.split(",")), context=a.context, chunks=chunks,
                         steps=a.steps, warmup=a.warmup, kernels=a.kernels, only=a.only)))


if __name__ == "__main__":
    main()

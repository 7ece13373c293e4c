"""Prefill and decode of a mixed stack (the Sikazen design) beside the closest other models of the framework at equal size.  No other model has all
three of its mixers, so there are two: the hyper-connected stack with one residual stream (windowed attention, linear attention with a decay per
key channel, full attention), and the multi-head latent attention stack with dense feed-forwards (rotated latent attention).  Same widths, heads,
window, latents, recurrent state, feed-forwards and number of layers.  bf16 weights, random, one GPU.

    python bench.py --config sikazen                                   # every size, all models, one JSON line
    python bench.py --config sikazen --sikazen-size medium
    python -m cuteafd_b200.bench.mixed_stack --size medium --kernels   # plus device time and share of the roofline per launch site

Timing as in `bench.latent_stack`.  Of three layers, one is rotated latent attention with sinks, one HGRN2, one windowed attention with a pooled key for
every 16 tokens in front of the window; every layer ends with the second token table.
"""
from __future__ import annotations

import argparse
import functools
import gc
import json

import torch

from ..config import AttentionSpec, ModelSpec, MoESpec, QuantSpec, sikazen_spec, vozetar_spec
from . import hyper_stack
from .hyper_stack import at_position
from .latent_stack import measure, peaks_used

# hidden, heads, key heads, dense feed-forward width, queries' latent, layers; windows of 2048, latents of 512, blocks of 16
SIZES = {"small": (2048, 16, 2, 6144, 768, 12), "medium": (4096, 32, 4, 12288, 1536, 6), "large": (8192, 64, 8, 24576, 1536, 6)}
MODELS = ("sikazen", "vozetar", "mla")
SIDE = 256


def specs(size: str) -> dict:
    hidden, heads, kv, ff, q_rank, layers = SIZES[size]
    ours = sikazen_spec(n_layers=layers, hidden=hidden, heads=heads, kv_heads=kv, ff=ff, q_rank=q_rank, rec_heads=hidden // 256, side=SIDE)
    mla = ModelSpec(name="mla-equal", family="deepseek_v3", vocab=ours.vocab, hidden=hidden, n_layers=layers, rms_eps=1e-5,
                    attn=AttentionSpec(kind="mla", n_heads=heads, n_kv_heads=heads, head_dim=192, q_lora_rank=q_rank, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128),
                    moe=MoESpec(n_experts=0, n_shared=0, top_k=1, first_dense=layers, dense_intermediate=ff), quant=QuantSpec(experts="bf16", dense="bf16", kv="bf16"))
    return {"sikazen": ours, "mla": mla,
            "vozetar": vozetar_spec(n_layers=layers, hidden=hidden, heads=heads, kv_heads=kv, ff=ff, rec_heads=hidden // 256, streams=1, mixers="GGA")}


def roofline(spec: ModelSpec, T: int, pairs: int, kv_rows: int, site: tuple, prefill: bool, peaks: dict, *, context: int, chunks: dict) -> tuple | None:
    """(label, ideal milliseconds of one launch) by what a launch has to compute and move; None = control work without a bound."""
    if spec.family == "vozetar":
        return hyper_stack.roofline(spec, T, pairs, kv_rows, site, prefill, peaks, context=context, chunks=chunks)
    W, H, ours = spec.hidden, spec.attn.n_heads, spec.family == "sikazen"
    lat = spec.attn
    rank, q_rank = lat.kv_lora_rank, lat.q_lora_rank
    tf, bw = peaks["bf16_tflops"] * 1e9, peaks["hbm_gbs"] * 1e6            # per millisecond
    lo = lambda ops, nbytes: max(ops / tf, nbytes / bw)
    seqs, ctx = (1, chunks[T]) if prefill else (T, context + 1)
    rows = seqs * ctx                                                       # cached rows of the step's sequences
    seen = sum(range(ctx - T + 1, ctx + 1)) if prefill else rows            # (query, key) pairs of a causal layer
    if site[0] == "gemm":
        _, form, sw, N, K = site
        if form == "grouped":
            return ("q -> latent" if K == lat.v_head_dim else "latent -> v", lo(2.0 * T * H * N * K, 2.0 * (H * N * K + T * H * (N + K))))
        if N == spec.vocab:
            return ("head", lo(2.0 * seqs * N * K, 2.0 * N * K + 4.0 * seqs * N))
        if prefill and K == rank and N == H * 256:
            return ("context -> keys, values", lo(2.0 * rows * N * K, 2.0 * (N * K + rows * (N + K))))
        mats = 2 if sw else 1
        label = ("ffn gate + up" if sw else "side gate" if ours and N == spec.side_dim else "side projection" if ours and K == spec.side_dim else "queries from their latent" if K == q_rank else
                 "latent: down projection" if N in (q_rank, rank + 64, q_rank + rank + 64) else "output projection (+ ffn down)" if N == W else "input projection")
        return (label, lo(2.0 * T * N * K * mats, 2.0 * (mats * N * K + T * (N + K))))
    n = site[0]
    if n in ("latent_attention", "mla_attention"):
        return ("attention (absorbed)", lo(2.0 * seen * H * (rank + 64 + rank), 2.0 * (rows * (rank + 64) + T * H * (2 * rank + 64))))
    if n in ("latent_prefill_attention", "mla_prefill_attention"):
        return ("attention (expanded)", lo(2.0 * seen * H * 320, 2.0 * (rows * (H * 256 + 64) + T * H * 320)))
    if n in ("latent_gather_ctx", "mla_gather_ctx"):
        return ("context gather", lo(0, 4.0 * rows * (rank + 64)))
    if n in ("latent_down", "mla_kv_prepare"):
        return ("latent: norms, rotation", lo(0, T * ((4.0 + 2.0) * (q_rank + rank + 64) if n == "latent_down" else 4.0 * (rank + 64))))
    if n in ("latent_split", "mla_q_split"):
        return ("latent: query heads", lo(0, 4.0 * T * H * 192))
    if n == "head_to_token_major":
        return ("head-major -> token-major", lo(0, 4.0 * T * H * 128))
    if n == "norm_rows":                                                    # both launches behind a layer, and the embedding
        return ("norm (+ residual)", lo(0, T * W * (4.0 + 4.0 + 2.0 + 2.0)))
    if n == "add_rmsnorm":
        return ("norm (+ residual)", lo(0, 4.0 * T * W))
    if n == "side_gate":
        return ("side gate: gelu, table", lo(0, T * SIDE * 8.0))
    if not ours:
        return None
    a = next(b.attn for b in spec.blocks if b.attn is not None and b.attn.kind == "conv_gqa")
    r = next(b.rec for b in spec.blocks if b.rec is not None)
    G, win, P = a.n_kv_heads, a.window, a.pool
    if n in ("window_attention", "window_prefill_attention"):
        keys = lambda p: min(p + 1, win) + max(0, p - win + 1) // P
        if prefill:
            q, c = sum(keys(p) for p in range(ctx - T, ctx)), min(ctx, T + win) + max(0, ctx - win) // P
        else:
            q = c = seqs * keys(context)
        return ("attention", lo(2.0 * q * H * 256, 2.0 * (c * G * 256 + T * H * 256)))
    if n == "conv_qkv":
        return ("queries, keys: conv, norm, rotation", lo(0, 2.0 * T * (a.conv_channels + (H + 2 * G) * 128)))
    if n == "pool_kv":
        return ("pooled blocks", lo(0, 2.0 * T * G * 256 * (1 + 1 / P)))
    if n == "decay_scan":
        d, dv = r.heads * r.dim, r.heads * r.vdim
        ops = 2.0 * T * r.heads * (64 * (r.dim + r.vdim) + 2 * r.dim * r.vdim) if prefill else 0
        return ("recurrence", lo(ops, 2.0 * T * (2 * d + 2 * dv) + 8.0 * seqs * r.heads * r.dim * r.vdim))
    return None


def run(sizes=tuple(SIZES), *, batches=(16, 64), context: int = 4096, chunks=((4096, 4096), (2048, 16384)), steps: int = 20, warmup: int = 3, kernels: bool = False,
        clocks=None, only: str = "") -> dict:
    peaks = peaks_used()
    out = {"bench": "sikazen", "peaks": peaks, "sizes": {}}
    if clocks is not None:
        clocks.start()
    for size in sizes:
        hidden, heads, kv, ff, q_rank, layers = SIZES[size]
        entry = {"shape": {"hidden": hidden, "heads": heads, "kv_heads": kv, "ff": ff, "q_rank": q_rank, "kv_rank": 512, "layers": layers, "window": 2048, "pool": 16, "side": SIDE}}
        for name, spec in specs(size).items():
            if only and name != only:
                continue
            entry[name] = measure(spec, batches=batches, context=context, chunks=chunks, steps=steps, warmup=warmup, kernels=kernels, peaks=peaks,
                                  roofline=functools.partial(roofline, context=context, chunks=dict(chunks)), at_position=at_position)
            gc.collect()
            torch.cuda.empty_cache()
        out["sizes"][size] = entry
    if clocks is not None:
        out["clocks"] = clocks.stop()
    return out


def bench_line(args, clocks) -> dict:
    """The `bench.py --config sikazen` line: decode throughput of the largest measured size, everything else under `results`."""
    sizes = tuple(SIZES) if args.sikazen_size == "all" else (args.sikazen_size,)
    res = run(sizes, steps=args.steps, warmup=args.warmup, clocks=clocks)
    size = sizes[-1]
    d = res["sizes"][size]["sikazen"]["decode"][-1]
    return {"metric": "decode_tokens_per_s", "value": d["tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
            "ms_per_step": d["ms_per_step"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16 operands, fp32 residual and recurrent state",
            "data": "synthetic token ids, random-init weights, context keys, values and latents random-filled",
            "config": {"model": f"{specs(size)['sikazen'].name} ({size})", "global_batch": d["batch"], "seq_len": d["context"], "parallelism": "single",
                       "l2": "weights far larger than L2; no flush needed"},
            "clocks": res.pop("clocks", None), "gpu_launches": sum(s["sikazen"]["gpu_launches"] for s in res["sizes"].values()), "results": res}


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--size", default="all", choices=["all", *SIZES])
    ap.add_argument("--steps", type=int, default=20); ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--context", type=int, default=4096); ap.add_argument("--batches", default="16,64")
    ap.add_argument("--chunks", default="4096:4096,2048:16384", help="prefill chunk:context pairs")
    ap.add_argument("--kernels", action="store_true"); ap.add_argument("--only", default="", choices=["", *MODELS])
    a = ap.parse_args()
    chunks = tuple(tuple(int(x) for x in c.split(":")) for c in a.chunks.split(",") if c)
    print(json.dumps(run(tuple(SIZES) if a.size == "all" else (a.size,), batches=tuple(int(b) for b in a.batches.split(",") if b), context=a.context, chunks=chunks,
                         steps=a.steps, warmup=a.warmup, kernels=a.kernels, only=a.only)))


if __name__ == "__main__":
    main()

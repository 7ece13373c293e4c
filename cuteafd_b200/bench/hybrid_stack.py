"""Prefill and decode of a hybrid recurrent / windowed-attention stack (the Tudilix design) beside the closest other model of the framework at
equal size: the hybrid stack with gated delta-rule layers (`engine.engine`), same widths, attention heads, window, feed-forward widths and
number of layers, two recurrent layers for every attention layer on both sides.  bf16 weights, random, one GPU.

    python bench.py --config tudilix                                   # every size, both models, one JSON line
    python bench.py --config tudilix --tudilix-size medium
    python -m cuteafd_b200.bench.hybrid_stack --size medium --kernels  # plus device time and share of the roofline per launch site

Timing as in `bench.latent_stack`.  Prompts of the other model run its recurrence token by token (it has no chunked form).
"""
from __future__ import annotations

import argparse
import gc
import json

import torch

from ..config import AttentionSpec, ModelSpec, MoESpec, QuantSpec, tudilix_spec
from .latent_stack import measure, peaks_used

# hidden (= recurrent width), heads, key heads, feed-forward width, channel blocks, layers; windows of 2048
SIZES = {"small": (2048, 16, 2, 6144, 8, 12), "medium": (4096, 32, 4, 12288, 16, 6), "large": (8192, 64, 8, 24576, 32, 6)}


def specs(size: str) -> tuple[ModelSpec, ModelSpec]:
    hidden, heads, kv, ff, blocks, layers = SIZES[size]
    ours = tudilix_spec(n_layers=layers, hidden=hidden, heads=heads, kv_heads=kv, ff=ff, blocks=blocks, ffn_everywhere=True)
    gdn = ModelSpec(name="gdn-equal", family="hybrid_linear", vocab=ours.vocab, hidden=hidden, n_layers=layers, rms_eps=1e-6,
                    attn=AttentionSpec(kind="gqa", n_heads=heads, n_kv_heads=kv, head_dim=128, rope_interleaved=False, qk_norm=True, window=ours.attn.window,
                                       linear_every=3, linear_k_heads=hidden // 256, linear_v_heads=hidden // 128),
                    moe=MoESpec(n_experts=0, n_shared=0, first_dense=layers, dense_intermediate=ff), quant=QuantSpec(experts="bf16", dense="bf16", kv="bf16"))
    return ours, gdn


def roofline(spec: ModelSpec, T: int, pairs: int, kv_rows: int, site: tuple, prefill: bool, peaks: dict) -> tuple | None:
    """(label, ideal milliseconds of one launch) by what a launch has to compute and move; None = control work without a bound."""
    a, W = spec.attn, spec.hidden
    H, G = a.n_heads, a.n_kv_heads
    tf, bw = peaks["bf16_tflops"] * 1e9, peaks["hbm_gbs"] * 1e6            # per millisecond
    lo = lambda ops, nbytes: max(ops / tf, nbytes / bw)
    if spec.stack:
        r = next(b.rec for b in spec.blocks if b.rec is not None)
        C, sq, ff = r.width, r.width // r.blocks, next(b.ffn.intermediate for b in spec.blocks if b.ffn is not None)
    else:
        Hk, Hv, ff = a.linear_k_heads, a.linear_v_heads, spec.moe.dense_intermediate
    seqs = T if not prefill else 1
    if site[0] == "gemm":
        _, form, sw, N, K = site
        if form == "grouped":
            return ("recurrence gates", lo(2.0 * T * C * 2 * sq, 4.0 * C * sq + T * C * (2.0 + 8.0)))
        if N == spec.vocab:
            return ("head", lo(2.0 * seqs * N * K, 2.0 * N * K + 4.0 * seqs * N))
        if sw:
            return ("ffn gate + up", lo(4.0 * T * N * K, 2.0 * (2 * N * K + T * (N + K))))
        if K == ff:
            return ("ffn down", lo(2.0 * T * N * K, 2.0 * (N * K + T * (N + K))))
        ideal = lo(2.0 * T * N * K, 2.0 * (N * K + T * (N + K)))
        return ("output projection" if N == W else "input projection", ideal)
    n = site[0]
    if n in ("window_attention", "window_prefill_attention", "paged_attention_tc", "gqa_prefill_attention"):
        return ("attention", lo(2.0 * pairs * H * 256, 2.0 * (kv_rows * G * 256 + T * H * 256)))
    if n == "conv_qkv":          # the average of layers with and without keys of their own
        return ("queries, keys: conv, norm, rotation", lo(0, 4.0 * T * (H + G) * 128))
    if n == "qk_norm_rope_kvwrite":
        return ("queries, keys: conv, norm, rotation", lo(0, 4.0 * T * (H + 2 * G) * 128))
    if n == "rglru_conv":
        return ("recurrence conv", lo(0, 4.0 * T * C))
    if n == "short_conv4":
        return ("recurrence conv", lo(0, 4.0 * T * (2 * Hk + Hv) * 128))
    if n == "lru_scan":
        return ("recurrence", lo(0, 14.0 * T * C + 8.0 * seqs * C))
    if n == "gated_delta_step":
        return ("recurrence", lo(0, 8.0 * T * Hv * 128 + 8.0 * seqs * Hv * 128 * 128))
    if n == "linear_prepare":
        return ("recurrence: head norms, gates", lo(0, 2.0 * T * ((2 * Hk + Hv) + 3 * Hv) * 128))
    if n == "gated_rmsnorm":
        return ("recurrence: output norm, gate", lo(0, 6.0 * T * Hv * 128))
    if n == "norm_rows":
        return ("norm (+ residual)", lo(0, 12.0 * T * W))
    if n == "add_rmsnorm":
        return ("norm (+ residual)", lo(0, 4.0 * T * W))
    return None


def run(sizes=tuple(SIZES), *, batches=(16, 64), context: int = 4096, chunks=((4096, 4096), (2048, 16384)), steps: int = 20, warmup: int = 3, kernels: bool = False,
        clocks=None, only: str = "") -> dict:
    peaks = peaks_used()
    out = {"bench": "tudilix", "peaks": peaks, "sizes": {}}
    if clocks is not None:
        clocks.start()
    for size in sizes:
        hidden, heads, kv, ff, blocks, layers = SIZES[size]
        entry = {"shape": {"hidden": hidden, "heads": heads, "kv_heads": kv, "ff": ff, "blocks": blocks, "layers": layers, "window": 2048}}
        for name, spec in zip(("tudilix", "gdn"), specs(size)):
            if only and name != only:
                continue
            entry[name] = measure(spec, batches=batches, context=context, chunks=chunks, steps=steps, warmup=warmup, kernels=kernels, peaks=peaks, roofline=roofline)
            gc.collect()
            torch.cuda.empty_cache()
        out["sizes"][size] = entry
    if clocks is not None:
        out["clocks"] = clocks.stop()
    return out


def bench_line(args, clocks) -> dict:
    """The `bench.py --config tudilix` line: decode throughput of the largest measured size, everything else under `results`."""
    sizes = tuple(SIZES) if args.tudilix_size == "all" else (args.tudilix_size,)
    res = run(sizes, steps=args.steps, warmup=args.warmup, clocks=clocks)
    size = sizes[-1]
    d = res["sizes"][size]["tudilix"]["decode"][-1]
    ours, _ = specs(size)
    return {"metric": "decode_tokens_per_s", "value": d["tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
            "ms_per_step": d["ms_per_step"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16 operands, fp32 residual and recurrent state",
            "data": "synthetic token ids, random-init weights, context keys and values random-filled",
            "config": {"model": f"{ours.name} ({size})", "global_batch": d["batch"], "seq_len": d["context"], "parallelism": "single",
                       "l2": "weights far larger than L2; no flush needed"},
            "clocks": res.pop("clocks", None), "gpu_launches": sum(s["tudilix"]["gpu_launches"] for s in res["sizes"].values()), "results": res}


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--size", default="all", choices=["all", *SIZES])
    ap.add_argument("--steps", type=int, default=20); ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--context", type=int, default=4096); ap.add_argument("--batches", default="16,64")
    ap.add_argument("--chunks", default="4096:4096,2048:16384", help="prefill chunk:context pairs")
    ap.add_argument("--kernels", action="store_true"); ap.add_argument("--only", default="", choices=["", "tudilix", "gdn"])
    a = ap.parse_args()
    chunks = tuple(tuple(int(x) for x in c.split(":")) for c in a.chunks.split(",") if c)
    print(json.dumps(run(tuple(SIZES) if a.size == "all" else (a.size,), batches=tuple(int(b) for b in a.batches.split(",") if b), context=a.context, chunks=chunks,
                         steps=a.steps, warmup=a.warmup, kernels=a.kernels, only=a.only)))


if __name__ == "__main__":
    main()

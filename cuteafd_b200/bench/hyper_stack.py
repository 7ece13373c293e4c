"""Prefill and decode of a hyper-connected stack with side-by-side mixers (the Vozetar design) beside the closest other model of the framework at
equal size: the hybrid stack with delta-rule layers of one decay per key channel (`engine.engine`, KDA), same widths, attention heads, window,
recurrent state per layer, feed-forwards and number of layers.  bf16 weights, random, one GPU.

    python bench.py --config vozetar                                   # every size, both models, one JSON line
    python bench.py --config vozetar --vozetar-size medium
    python -m cuteafd_b200.bench.hyper_stack --size medium --kernels   # plus device time and share of the roofline per launch site

Timing as in `bench.latent_stack`.  Of three layers, two run two mixers side by side (attention beside retention, attention beside gated linear
attention), the third full attention alone; the other model alternates delta-rule and attention layers and runs prompts through its recurrence
token by token (it has no chunked form).
"""
from __future__ import annotations

import argparse
import functools
import gc
import json

import torch

from ..config import AttentionSpec, ModelSpec, MoESpec, QuantSpec, vozetar_spec
from .latent_stack import measure, peaks_used

# hidden, heads, key heads, dense feed-forward width, experts (0: dense; else of the width below, 8 per token and a shared one), layers; windows of 2048
SIZES = {"small": (2048, 16, 2, 6144, 0, 12), "medium": (4096, 32, 4, 12288, 0, 6), "moe": (4096, 32, 4, 0, 64, 6), "large": (8192, 64, 8, 24576, 0, 6)}
EXPERT_FF, STREAMS = 1536, 4


def specs(size: str) -> tuple[ModelSpec, ModelSpec]:
    hidden, heads, kv, ff, experts, layers = SIZES[size]
    ours = vozetar_spec(n_layers=layers, hidden=hidden, heads=heads, kv_heads=kv, ff=ff, rec_heads=hidden // 256, experts=experts, expert_ff=EXPERT_FF, streams=STREAMS, moe_every=1)
    moe = ours.moe if experts else MoESpec(n_experts=0, n_shared=0, first_dense=layers, dense_intermediate=ff)
    kda = ModelSpec(name="kda-equal", family="hybrid_linear", vocab=ours.vocab, hidden=hidden, n_layers=layers, rms_eps=1e-5,
                    attn=AttentionSpec(kind="gqa", n_heads=heads, n_kv_heads=kv, head_dim=128, rope_interleaved=False, qk_norm=True, window=ours.attn.window,
                                       linear_every=2, linear_k_heads=hidden // 256, linear_v_heads=hidden // 128, linear_per_channel=True),
                    moe=moe, quant=QuantSpec(experts="bf16", dense="bf16", kv="bf16"))
    return ours, kda


def at_position(eng, pos: int):
    """The linear mixers' states sit in front of position `pos` (their contents are whatever they are)."""
    for s in getattr(eng, "states", None) or []:
        if s is not None:
            s[1].copy_(torch.tensor([pos - 1, -1], dtype=torch.int32, device=eng.device).expand_as(s[1]))


def roofline(spec: ModelSpec, T: int, pairs: int, kv_rows: int, site: tuple, prefill: bool, peaks: dict, *, context: int, chunks: dict) -> tuple | None:
    """(label, ideal milliseconds of one launch) by what a launch has to compute and move; None = control work without a bound.  Launches that
    differ from layer to layer count as the average of their layers."""
    a, m, W = spec.attn, spec.moe, spec.hidden
    H, G, k = a.n_heads, a.n_kv_heads, m.top_k
    tf, bw = peaks["bf16_tflops"] * 1e9, peaks["hbm_gbs"] * 1e6            # per millisecond
    lo = lambda ops, nbytes: max(ops / tf, nbytes / bw)
    seqs = T if not prefill else 1
    ours = bool(spec.stack)
    blocks = spec.blocks
    mean = lambda f, of: sum(f(b) for b in of) / len(of)
    recs = [b for b in blocks if b.rec is not None]
    if ours:
        dense = max((b.ffn.intermediate for b in blocks if b.ffn is not None), default=0)
    else:
        Hk, Hv, dense = a.linear_k_heads, a.linear_v_heads, 0 if m.n_experts else m.dense_intermediate
    if site[0] == "gemm":
        _, form, sw, N, K = site
        if form == "grouped":
            act, mats = min(m.n_experts, T * k), 2 if sw else 1
            return ("experts up" if N == m.intermediate else "experts down", lo(2.0 * T * k * N * K * mats, 2.0 * (act * N * K * mats + T * k * (N + K))))
        if N == spec.vocab:
            return ("head", lo(2.0 * seqs * N * K, 2.0 * N * K + 4.0 * seqs * N))
        if m.n_experts and N == m.n_experts:
            return ("router logits", lo(2.0 * T * N * K, 2.0 * N * K + T * (2.0 * K + 4.0 * N)))
        if sw:
            return ("ffn gate + up", lo(4.0 * T * N * K, 2.0 * (2 * N * K + T * (N + K))))
        if K == dense or (m.n_experts and K == m.shared_inter):
            return ("ffn down", lo(2.0 * T * N * K, 2.0 * (N * K + T * (N + K))))
        return ("output projection" if N == W else "input projection", lo(2.0 * T * N * K, 2.0 * (N * K + T * (N + K))))
    n = site[0]
    if n in ("window_attention", "window_prefill_attention", "paged_attention_tc", "gqa_prefill_attention"):
        if not ours:
            return ("attention", lo(2.0 * pairs * H * 256, 2.0 * (kv_rows * G * 256 + T * H * 256)))
        ctx = chunks[T] if prefill else context
        full = (sum(range(ctx - T + 1, ctx + 1)), ctx) if prefill else (T * (ctx + 1), T * (ctx + 1))

        def one(b):
            seen, rows = (pairs, kv_rows) if b.attn.window else full
            return lo(2.0 * seen * H * 256, 2.0 * (rows * G * 256 + T * (H * 256 + b.attn.gate_width)))
        return ("attention", mean(one, blocks))
    if n == "conv_qkv":
        return ("queries, keys: conv, norm, rotation", mean(lambda b: lo(0, 2.0 * T * (b.attn.conv_channels + (H + 2 * G) * 128)), blocks))
    if n == "qk_norm_rope_kvwrite":
        return ("queries, keys: conv, norm, rotation", lo(0, 4.0 * T * (H + 2 * G) * 128))
    if n == "decay_scan":
        def rec(b):
            r = b.rec
            d, dv = r.heads * r.dim, r.heads * r.vdim
            ops = 2.0 * T * r.heads * (64 * (r.dim + r.vdim) + 2 * r.dim * r.vdim) if prefill else 0
            return lo(ops, 2.0 * T * (2 * d + 3 * dv) + 8.0 * seqs * r.heads * r.dim * r.vdim + (4.0 * d * r.rank if r.rank else 0))
        return ("recurrence", mean(rec, recs))
    if n == "gated_delta_step":
        return ("recurrence", lo(0, 2.0 * T * Hv * 128 * 6 + 8.0 * seqs * Hv * 128 * 128))
    if n == "short_conv4":
        return ("recurrence: conv", lo(0, 4.0 * T * (2 * Hk + Hv) * 128))
    if n == "linear_prepare":
        return ("recurrence: head norms, gates", lo(0, T * 128 * (2.0 * (2 * Hk + Hv) + 4.0 * Hv + 10.0 * Hv)))
    if n == "gated_rmsnorm":
        return ("recurrence: output norm, gate", lo(0, 6.0 * T * Hv * 128))
    if n == "hyper_rows":
        return ("norm (+ residual)", lo(0, T * W * (8.0 * spec.streams + 5.0 + (k if m.n_experts else 0))))        # both boundaries of a layer
    if n in ("moe_combine", "moe_combine_norm"):
        return ("combine (+ norm)", lo(0, T * W * (2.0 * k + 8)))
    if n == "add_rmsnorm":
        return ("norm (+ residual)", lo(0, 4.0 * T * W))
    if n == "gather_rows":
        return ("expert gather", lo(0, 4.0 * T * k * W)) if m.n_experts else None
    if n == "router_logits":
        return ("router logits", lo(0, 2.0 * m.n_experts * W + T * (2.0 * W + 4.0 * m.n_experts)))
    return None


def run(sizes=tuple(SIZES), *, batches=(16, 64), context: int = 4096, chunks=((4096, 4096), (2048, 16384)), steps: int = 20, warmup: int = 3, kernels: bool = False,
        clocks=None, only: str = "") -> dict:
    peaks = peaks_used()
    out = {"bench": "vozetar", "peaks": peaks, "sizes": {}}
    if clocks is not None:
        clocks.start()
    for size in sizes:
        hidden, heads, kv, ff, experts, layers = SIZES[size]
        entry = {"shape": {"hidden": hidden, "heads": heads, "kv_heads": kv, "ff": ff, "experts": experts, "layers": layers, "window": 2048, "streams": STREAMS}}
        for name, spec in zip(("vozetar", "kda"), specs(size)):
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
    """The `bench.py --config vozetar` line: decode throughput of the largest measured size, everything else under `results`."""
    sizes = tuple(SIZES) if args.vozetar_size == "all" else (args.vozetar_size,)
    res = run(sizes, steps=args.steps, warmup=args.warmup, clocks=clocks)
    size = sizes[-1]
    d = res["sizes"][size]["vozetar"]["decode"][-1]
    ours, _ = specs(size)
    return {"metric": "decode_tokens_per_s", "value": d["tokens_per_s"], "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup,
            "ms_per_step": d["ms_per_step"], "higher_is_better": True, "scaling": "weak", "vs_baseline": None, "dtype": "bf16 operands, fp32 residual streams and recurrent state",
            "data": "synthetic token ids, random-init weights, context keys and values random-filled",
            "config": {"model": f"{ours.name} ({size})", "global_batch": d["batch"], "seq_len": d["context"], "parallelism": "single",
                       "l2": "weights far larger than L2; no flush needed"},
            "clocks": res.pop("clocks", None), "gpu_launches": sum(s["vozetar"]["gpu_launches"] for s in res["sizes"].values()), "results": res}


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--size", default="all", choices=["all", *SIZES])
    ap.add_argument("--steps", type=int, default=20); ap.add_argument("--warmup", type=int, default=3)
    ap.add_argument("--context", type=int, default=4096); ap.add_argument("--batches", default="16,64")
    ap.add_argument("--chunks", default="4096:4096,2048:16384", help="prefill chunk:context pairs")
    ap.add_argument("--kernels", action="store_true"); ap.add_argument("--only", default="", choices=["", "vozetar", "kda"])
    a = ap.parse_args()
    chunks = tuple(tuple(int(x) for x in c.split(":")) for c in a.chunks.split(",") if c)
    print(json.dumps(run(tuple(SIZES) if a.size == "all" else (a.size,), batches=tuple(int(b) for b in a.batches.split(",") if b), context=a.context, chunks=chunks,
                         steps=a.steps, warmup=a.warmup, kernels=a.kernels, only=a.only)))


if __name__ == "__main__":
    main()

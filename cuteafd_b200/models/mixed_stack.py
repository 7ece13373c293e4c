"""Device weights of mixed stacks (the Sikazen design) in the forms the kernels consume.

A layer's mixer and feed-forward read the same unit-normed row, each times a number of its own; the numbers are output factors of the products
that read the row (`TcWeight.alpha`), so one operand row serves both and no weight is rounded a second time.  Everything of the mixer that
reads the row is one matrix (`w_in`, segments on 16-byte boundaries: `MixedLayer.columns`).  Mixer and feed-forward are added, so they share
one output projection over both operands side by side (`wo`: [mixer | feed-forward]).

Widths are padded so that every operand row starts on a 16-byte boundary (multiples of 8; latents, per-head query widths and rotated parts to
whole 64-element chunks); pads are zero in the weights, so they stay zero in the activations.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..config import BlockSpec, ModelSpec
from ..ops import KIND_BF16, KIND_F32, TcWeight
from .hybrid_stack import HybridWeights, rope_tables
from .hyper_stack import HyperLayer, place
from .latent_stack import StackLayer, _pad, stack_kind, up


@dataclass
class MixedLayer(HyperLayer, StackLayer):
    """Attention uses `w_in` and `qkv_b`; latent attention `w_in`, `q_norm` (of the queries' latent), `kv_norm`, `w_uq`, `w_uk_t`, `w_uv`, `sink`; HGRN2
    `w_in`, `forget_b`, `lower`, `lin_norm`; the feed-forward `ws_gate`, `ws_up` and the last columns of `wo`."""
    w_uq: TcWeight | None = None
    forget_b: torch.Tensor | None = None    # [heads * dim] bias and lower bound of the forget gate
    lower: torch.Tensor | None = None
    side_gate: TcWeight | None = None       # [side_pad, hidden_pad], [hidden_pad, side_pad]
    side_proj: TcWeight | None = None
    side_norm: torch.Tensor | None = None


@dataclass
class MixedWeights(HybridWeights):
    side: torch.Tensor | None = None        # [vocab, layers * side_dim] bf16

    def nbytes(self) -> int:
        return super().nbytes() + (self.side.numel() * 2 if self.side is not None else 0)


def input_segments(b: BlockSpec) -> list[tuple[str, int]]:
    """Segments of a layer's input projection and their rows."""
    a, r = b.attn, b.rec
    if r is not None:
        return [("rq", r.heads * r.dim), ("rf", r.heads * r.dim), ("rv", r.heads * r.vdim)]
    if a.kind == "latent":
        return [("dq", a.q_lora_rank), ("dkv", a.kv_lora_rank + a.rope_dims)]
    return [("qkv", a.conv_channels)]


def mixer_width(b: BlockSpec) -> int:
    """Values per token that a mixer hands to its output projection."""
    return b.rec.heads * b.rec.vdim if b.rec is not None else b.attn.n_heads * b.attn.v_head_dim


def check_blocks(spec: ModelSpec):
    if spec.loop is not None and spec.loop.entry != "add":
        raise ValueError("mixed stacks open a pass of their loop by adding the embedding output")
    for i, b in enumerate(spec.blocks):
        a, r = b.attn, b.rec
        if b.moe is not None or (a is None) == (r is None) or (r is not None and r.kind != "hgrn2") or (a is not None and a.kind not in ("conv_gqa", "latent")):
            raise ValueError(f"layer {i}: mixed stacks have attention, latent attention or HGRN2, and dense feed-forwards")
        if r is not None and (r.dim > 512 or r.vdim > 1024):
            raise ValueError(f"layer {i}: recurrent heads of up to 512 x 1024 (got {r.dim} x {r.vdim})")
        if a is not None and a.kind == "latent" and (a.q_lora_rank < 1 or a.kv_lora_rank > 1024):
            raise ValueError(f"layer {i}: queries through a latent, keys and values through one of up to 1024 values (got {a.q_lora_rank} / {a.kv_lora_rank})")
        if a is not None and a.kind == "conv_gqa" and (a.conv_taps or max(a.head_dim, a.v_head_dim) > 256):
            raise ValueError(f"layer {i}: heads of up to 256 dimensions without convolutions (got {a.head_dim} / {a.v_head_dim})")


def mixed_weights_from_masters(spec: ModelSpec, masters: dict, device) -> MixedWeights:
    """`masters` as `loader.stack_checkpoint.read_mixed_masters` returns them (any floating dtype)."""
    kind = stack_kind(spec)
    W, Wp, sd = spec.hidden, up(spec.hidden, 8), spec.side_dim
    vec = lambda t, n: _pad(t.float().reshape(-1), n).to(device).contiguous()
    f32 = lambda t: t.float().to(device).contiguous()

    def mat(t, *shape, alpha: float | None = None) -> TcWeight:
        w = TcWeight.from_master(_pad(t, *shape), kind, device)
        if alpha is not None:
            w.alpha = torch.full((w.G,), alpha, dtype=torch.float32, device=device)
        return w

    def layer(b, lw) -> MixedLayer:
        a, r = b.attn, b.rec
        cols, rows = place(input_segments(b))
        parts = {n: lw.get(n) for n in ("rq", "rf", "rv", "dq", "dkv")}
        if "qkv" in cols:
            parts["qkv"] = torch.cat([lw[f"w{k}"] for k in ("q", "k", "v")])
        w = torch.zeros(rows, W, dtype=torch.float32 if kind == "f32" else torch.bfloat16)
        for name, (at, n) in cols.items():
            w[at:at + n] = parts[name]
        K1, wo = up(mixer_width(b), 8), lw["wo"]
        if b.ffn is not None:
            f8 = up(b.ffn.intermediate, 8)
            wo = torch.cat([_pad(wo, W, K1), _pad(lw["ws_down"], W, f8)], 1)
        out = MixedLayer(attn_norm=None, ffn_norm=None, wqkv=None, wo=mat(wo, Wp, up(wo.shape[1], 8)), columns=cols, w_in=mat(w, rows, Wp, alpha=lw["norm1"]))
        if r is not None:
            out.forget_b, out.lower, out.lin_norm = f32(lw["f_b"]), f32(lw["lower"]), f32(lw["r_norm"])
        elif a.kind == "latent":
            H, d, dv, rk = a.n_heads, a.head_dim, a.v_head_dim, a.kv_lora_rank
            rp, dp = up(rk, 64), up(d, 64)
            out.q_norm, out.kv_norm, out.sink = f32(lw["dq_norm"]), f32(lw["dkv_norm"]), f32(lw["sink"])
            out.w_uq = mat(lw["uq"], lw["uq"].shape[0], up(a.q_lora_rank, 8))
            out.w_uk_t = TcWeight.from_master(_pad(lw["w_uk"].reshape(H, d, rk).transpose(1, 2), H, rp, dp), kind, device)
            out.w_uv = mat(lw["w_uv"].reshape(H, dv, rk), H, dv, rp)
        else:
            out.qkv_b = f32(torch.cat([lw[f"{k}_b"] for k in ("q", "k", "v")]))
        if b.ffn is not None:
            out.ws_gate, out.ws_up = mat(lw["ws_gate"], f8, Wp, alpha=lw["norm2"]), mat(lw["ws_up"], f8, Wp, alpha=lw["norm2"])
        if sd:
            s8 = up(sd, 8)
            out.side_gate, out.side_proj, out.side_norm = mat(lw["side_gate"], s8, Wp), mat(lw["side_proj"], Wp, s8), vec(lw["side_norm"], Wp)
        return out

    check_blocks(spec)
    mw = MixedWeights(spec=spec, embed=_pad(masters["embed"].to(torch.bfloat16), spec.vocab, Wp).to(device).contiguous(), final_norm=None,
                      lm_head=mat(masters["lm_head"], spec.vocab, Wp, alpha=masters["final_norm"]), rope=rope_tables(spec, device),
                      side=masters["side"].to(torch.bfloat16).to(device).contiguous() if sd else None)
    mw.layers = [layer(b, lw) for b, lw in zip(spec.blocks, masters["layers"])]
    mw.layer_map = list(range(spec.n_layers))
    return mw


def mixed_weights_random(spec: ModelSpec, device, seed: int = 1) -> MixedWeights:
    """Random weights directly on the device (benchmarks of real layer sizes)."""
    kind, W, sd = stack_kind(spec), spec.hidden, spec.side_dim
    if W % 8:
        raise ValueError("random weights: the residual width must be a multiple of 8")
    check_blocks(spec)
    gen = torch.Generator(device=device).manual_seed(seed)
    nrm = lambda *s, std: torch.empty(*s, device=device).normal_(0, std, generator=gen)
    ones = lambda n: torch.ones(n, dtype=torch.float32, device=device)

    def R(G, N, K, std=None, keep=None, alpha=False):
        """Random [G, N, K] whose pads beyond `keep` = (rows, columns) are zero."""
        data = torch.empty(G, N, K, dtype=torch.bfloat16 if kind == "bf16" else torch.float32, device=device).normal_(0, std or K ** -0.5, generator=gen)
        if keep:
            data[:, keep[0]:] = 0
            data[:, :, keep[1]:] = 0
        w = TcWeight(KIND_BF16, G, N, K, data, ops.encode_tmap(data, 128)) if kind == "bf16" else TcWeight(KIND_F32, G, N, K, data, None)
        if alpha:
            w.alpha = ones(G)
        return w

    def layer(i, b) -> MixedLayer:
        a, r = b.attn, b.rec
        cols, rows = place(input_segments(b))
        K1 = up(mixer_width(b), 8)
        f8 = up(b.ffn.intermediate, 8) if b.ffn is not None else 0
        wo = R(1, W, K1 + f8)
        wo.data[:, :, mixer_width(b):K1] = 0
        out = MixedLayer(attn_norm=None, ffn_norm=None, wqkv=None, wo=wo, columns=cols, w_in=R(1, rows, W, alpha=True))
        if r is not None:       # lower bounds rise from 0 in the first layer towards 1 in the last
            out.forget_b, out.lower, out.lin_norm = nrm(r.heads * r.dim, std=1.0) + 2.0, ones(r.heads * r.dim) * (i / spec.n_layers), ones(r.vdim)
        elif a.kind == "latent":
            H, d, dv, rk = a.n_heads, a.head_dim, a.v_head_dim, a.kv_lora_rank
            rp, dp = up(rk, 64), up(d, 64)
            out.q_norm, out.kv_norm, out.sink = ones(a.q_lora_rank), ones(rk), nrm(H, std=1.0)
            out.w_uq = R(1, H * (d + a.rope_dims), up(a.q_lora_rank, 8), keep=(H * (d + a.rope_dims), a.q_lora_rank))
            out.w_uk_t, out.w_uv = R(H, rp, dp, std=rk ** -0.5, keep=(rk, d)), R(H, dv, rp, std=rk ** -0.5, keep=(dv, rk))
        else:
            out.qkv_b = nrm(a.conv_channels, std=0.1)
        if b.ffn is not None:
            ff = b.ffn.intermediate
            out.ws_gate, out.ws_up = R(1, f8, W, keep=(ff, W), alpha=True), R(1, f8, W, keep=(ff, W), alpha=True)
        if sd:
            s8 = up(sd, 8)
            out.side_gate, out.side_proj, out.side_norm = R(1, s8, W, keep=(sd, W)), R(1, W, s8, keep=(W, sd)), ones(W)
        return out

    mw = MixedWeights(spec=spec, embed=nrm(spec.vocab, W, std=spec.embed_scale ** -1).to(torch.bfloat16), final_norm=None, lm_head=R(1, spec.vocab, W, alpha=True), rope=rope_tables(spec, device),
                      side=nrm(spec.vocab, spec.n_layers * sd, std=1.0).to(torch.bfloat16) if sd else None)
    mw.layers = [layer(i, b) for i, b in enumerate(spec.blocks)]
    mw.layer_map = list(range(spec.n_layers))
    return mw

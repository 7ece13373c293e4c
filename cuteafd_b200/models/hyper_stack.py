"""Device weights of hyper-connected stacks with side-by-side mixers (the Vozetar design) in the forms the kernels consume.

Everything that reads a layer's normalised row is one matrix (`w_in`): queries, keys and values of the attention, its output gate, then - where
a linear mixer runs beside it - that one's queries, keys, values, output gate and low-rank decay input, each segment starting on a 16-byte
boundary (`HyperLayer.columns`).  Two mixers whose outputs are simply added share one output projection over both operands side by side; mixers
whose outputs are normalised first keep one each.

Widths are padded so that every operand row starts on a 16-byte boundary (multiples of 8); pads are zero in the weights, so they stay
zero in the activations.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..config import BlockSpec, ModelSpec
from ..ops import KIND_BF16, KIND_F32, TcWeight
from .hybrid_stack import HybridLayer, HybridWeights, rope_tables
from .latent_stack import _pad, stack_kind, up


@dataclass
class HyperLayer(HybridLayer):
    """Attention uses `w_in`, `conv`, `q_norm`, `k_norm`, `sink`, `wo`; a dense or shared feed-forward `ws_*`, routed experts `router` and `w_*`."""
    columns: dict | None = None             # segment of w_in -> (first row, rows)
    qkv_b: torch.Tensor | None = None       # biases of the attention's projections, in the order of their columns
    wo_b: torch.Tensor | None = None
    wo2: TcWeight | None = None             # the linear mixer's output projection where it is one of its own
    merge_norms: tuple | None = None        # gains of the norms behind both mixers
    lin_decay: torch.Tensor | None = None   # [heads] constant decays
    lin_a2: torch.Tensor | None = None      # [heads * dim, rank], [heads * dim]: logits of the per-channel decays
    lin_a2_b: torch.Tensor | None = None
    hc1: tuple | None = None                # (in [S], out [S], mix [S, S]) around the mixer and around the feed-forward
    hc2: tuple | None = None


@dataclass
class HyperWeights(HybridWeights):
    pair_rows: torch.Tensor | None = None   # [buckets + 1, hidden_pad] bf16

    def nbytes(self) -> int:
        return super().nbytes() + (self.pair_rows.numel() * 2 if self.pair_rows is not None else 0)


def input_segments(b: BlockSpec, rank: int) -> list[tuple[str, int]]:
    """Segments of a layer's input projection and their rows."""
    a, r = b.attn, b.rec
    out = [("qkv", a.conv_channels)] + ([("gate", a.gate_width)] if a.out_gate else [])
    if r is not None:
        out += [("rq", r.heads * r.dim), ("rk", r.heads * r.dim), ("rv", r.heads * r.vdim), ("rg", r.heads * r.vdim)] + ([("a1", rank)] if r.kind == "gla" else [])
    return out


def place(segments: list[tuple[str, int]]) -> tuple[dict, int]:
    """(segment -> (first row, rows), rows in all), every segment starting on a multiple of 8."""
    at, cols = 0, {}
    for name, n in segments:
        cols[name] = (at, n)
        at += up(n, 8)
    return cols, at


def check_blocks(spec: ModelSpec):
    for i, b in enumerate(spec.blocks):
        a, r, m = b.attn, b.rec, b.moe
        if a is None or (r is not None and r.kind not in ("retention", "gla")):
            raise ValueError(f"layer {i}: hyper-connected stacks have attention, alone or beside retention or gated linear attention")
        if not 0 <= a.conv_taps <= 16 or max(a.head_dim, a.v_head_dim) > 256:
            raise ValueError(f"layer {i}: convolutions of up to 16 taps and heads of up to 256 dimensions (got {a.conv_taps} and {a.head_dim} / {a.v_head_dim})")
        if r is not None and (r.dim > 512 or r.vdim > 1024):
            raise ValueError(f"layer {i}: recurrent heads of up to 512 x 1024 (got {r.dim} x {r.vdim})")
        if m is not None and (m.n_experts > 512 or m.top_k > 16 or m.n_group > 32):
            raise ValueError(f"layer {i}: at most 512 experts, 16 per token, 32 groups")
    if not 1 <= spec.streams <= 8:
        raise ValueError(f"1 to 8 residual streams (got {spec.streams})")


def hyper_weights_from_masters(spec: ModelSpec, masters: dict, device) -> HyperWeights:
    """`masters` as `loader.stack_checkpoint.read_hyper_masters` returns them (any floating dtype)."""
    kind = stack_kind(spec)
    W, Wp = spec.hidden, up(spec.hidden, 8)
    vec = lambda t, n: _pad(t.float().reshape(-1), n).to(device).contiguous()
    mat = lambda t, *shape: TcWeight.from_master(_pad(t, *shape), kind, device)
    f32 = lambda t: t.float().to(device).contiguous()
    table = lambda t: _pad(t.to(torch.bfloat16), t.shape[0], Wp).to(device).contiguous()

    def layer(b, lw) -> HyperLayer:
        a, r, m = b.attn, b.rec, b.moe
        qkv = ("q", "k") if a.values_are_keys else ("q", "k", "v")
        parts = {"qkv": torch.cat([lw[f"w{k}"] for k in qkv]), "gate": lw.get("wg")}
        if r is not None:
            parts.update({n: lw.get(n) for n in ("rq", "rk", "rv", "rg", "a1")})
        cols, rows = place(input_segments(b, lw["a1"].shape[0] if "a1" in lw else 0))
        w = torch.zeros(rows, W, dtype=torch.float32 if kind == "f32" else torch.bfloat16)
        for name, (at, n) in cols.items():
            w[at:at + n] = parts[name]
        K1 = up(a.n_heads * a.v_head_dim, 8)
        wo, wo2 = lw["wo"], None
        if r is not None:
            K2 = up(r.heads * r.vdim, 8)
            if b.merge_norm:
                wo2 = mat(lw["r_o"], Wp, K2)
            else:
                wo = torch.cat([_pad(wo, W, K1), _pad(lw["r_o"], W, K2)], 1)
        out = HyperLayer(attn_norm=vec(lw["norm1"], Wp), ffn_norm=None, wqkv=None, wo=mat(wo, Wp, up(wo.shape[1], 8)), columns=cols, w_in=mat(w, rows, Wp), wo2=wo2,
                         hc1=tuple(f32(t) for t in lw["hc1"]))
        if a.conv_taps:
            out.conv = f32(torch.cat([lw[f"{k}_conv"] for k in qkv]).float().T)
        if a.qkv_bias:
            out.qkv_b = f32(torch.cat([lw[f"{k}_b"] for k in qkv]))
        if a.out_bias:
            out.wo_b = vec(lw["o_b"], Wp)
        if a.sink:
            out.sink = f32(lw["sink"])
        if a.qk_norm_whole or a.qk_norm:
            out.q_norm, out.k_norm = f32(lw["q_norm"]), f32(lw["k_norm"])
        if r is not None and r.kind == "retention":
            out.lin_decay = torch.tensor(r.decay, dtype=torch.float32, device=device)
        elif r is not None:
            out.lin_a2, out.lin_a2_b, out.lin_norm = f32(lw["a2"]), f32(lw["a2_b"]), f32(lw["r_norm"])
        if b.merge_norm:
            out.merge_norms = tuple(vec(t, Wp) for t in lw["merge_norms"])
        if m is not None or b.ffn is not None:
            out.ffn_norm, out.hc2 = vec(lw["norm2"], Wp), tuple(f32(t) for t in lw["hc2"])
        dense = b.ffn.intermediate if b.ffn is not None else (m.shared_inter if m is not None and m.n_shared else 0)
        if dense:
            f8 = up(dense, 8)
            out.ws_gate, out.ws_up, out.ws_down = mat(lw["ws_gate"], f8, Wp), mat(lw["ws_up"], f8, Wp), mat(lw["ws_down"], Wp, f8)
        if m is not None:
            E, ff = m.n_experts, m.intermediate
            out.router = mat(lw["router"], E, Wp)
            out.w_gate, out.w_up, out.w_down = mat(lw["w_gate"], E, ff, Wp), mat(lw["w_up"], E, ff, Wp), mat(lw["w_down"], E, Wp, up(ff, 8))
        return out

    check_blocks(spec)
    hw = HyperWeights(spec=spec, embed=table(masters["embed"]), final_norm=vec(masters["final_norm"], Wp), lm_head=mat(masters["lm_head"], spec.vocab, Wp),
                      rope=rope_tables(spec, device), pair_rows=table(masters["pairs"]) if spec.pair_table is not None else None)
    hw.layers = [layer(b, lw) for b, lw in zip(spec.blocks, masters["layers"])]
    hw.layer_map = list(range(spec.n_layers))
    return hw


def hyper_weights_random(spec: ModelSpec, device, seed: int = 1) -> HyperWeights:
    """Random weights directly on the device (benchmarks of real layer sizes)."""
    kind, W, S = stack_kind(spec), spec.hidden, spec.streams
    if W % 8:
        raise ValueError("random weights: the residual width must be a multiple of 8")
    check_blocks(spec)
    gen = torch.Generator(device=device).manual_seed(seed)
    nrm = lambda *s, std: torch.empty(*s, device=device).normal_(0, std, generator=gen)
    ones = lambda n: torch.ones(n, dtype=torch.float32, device=device)

    def R(G, N, K, keep=None):
        """Random [G, N, K] whose pads beyond `keep` = (rows, columns) are zero."""
        data = torch.empty(G, N, K, dtype=torch.bfloat16 if kind == "bf16" else torch.float32, device=device).normal_(0, K ** -0.5, generator=gen)
        if keep:
            data[:, keep[0]:] = 0
            data[:, :, keep[1]:] = 0
        return TcWeight(KIND_BF16, G, N, K, data, ops.encode_tmap(data, 128)) if kind == "bf16" else TcWeight(KIND_F32, G, N, K, data, None)

    def constants() -> tuple:
        return (ones(S) / S, ones(S), 0.7 * torch.eye(S, device=device) + 0.3 / S)

    def layer(b) -> HyperLayer:
        a, r, m = b.attn, b.rec, b.moe
        cols, rows = place(input_segments(b, r.rank if r is not None else 0))
        H, G, K1 = a.n_heads, a.n_kv_heads, up(a.n_heads * a.v_head_dim, 8)
        K2 = up(r.heads * r.vdim, 8) if r is not None else 0
        out = HyperLayer(attn_norm=ones(W), ffn_norm=None, wqkv=None, wo=R(1, W, K1 if b.merge_norm else K1 + K2), columns=cols, w_in=R(1, rows, W), hc1=constants())
        out.conv = nrm(a.conv_taps, a.conv_channels, std=0.5) if a.conv_taps else None
        out.qkv_b = nrm(a.conv_channels, std=0.1) if a.qkv_bias else None
        out.wo_b = nrm(W, std=0.1) if a.out_bias else None
        out.sink = nrm(H, std=1.0) if a.sink else None
        if a.qk_norm_whole:
            out.q_norm, out.k_norm = ones(H * a.head_dim), ones(G * a.head_dim)
        if b.merge_norm:
            out.wo2, out.merge_norms = R(1, W, K2), (ones(W), ones(W))
        if r is not None and r.kind == "retention":
            out.lin_decay = torch.tensor(r.decay, dtype=torch.float32, device=device)
        elif r is not None:
            out.lin_a2, out.lin_a2_b, out.lin_norm = nrm(r.heads * r.dim, r.rank, std=r.rank ** -0.5), nrm(r.heads * r.dim, std=1.0), ones(r.vdim)
        if m is not None or b.ffn is not None:
            out.ffn_norm, out.hc2 = ones(W), constants()
        dense = b.ffn.intermediate if b.ffn is not None else (m.shared_inter if m is not None and m.n_shared else 0)
        if dense:
            f8 = up(dense, 8)
            out.ws_gate, out.ws_up, out.ws_down = R(1, f8, W, keep=(dense, W)), R(1, f8, W, keep=(dense, W)), R(1, W, f8, keep=(W, dense))
        if m is not None:
            E, ff = m.n_experts, m.intermediate
            out.router = R(1, E, W)
            out.w_gate, out.w_up, out.w_down = R(E, ff, W), R(E, ff, W), R(E, W, up(ff, 8), keep=(W, ff))
        return out

    pairs = nrm(spec.pair_table.buckets + 1, W, std=0.5).to(torch.bfloat16) if spec.pair_table is not None else None
    hw = HyperWeights(spec=spec, embed=nrm(spec.vocab, W, std=1.0).to(torch.bfloat16), final_norm=ones(W), lm_head=R(1, spec.vocab, W), rope=rope_tables(spec, device), pair_rows=pairs)
    hw.layers = [layer(b) for b in spec.blocks]
    hw.layer_map = list(range(spec.n_layers))
    return hw

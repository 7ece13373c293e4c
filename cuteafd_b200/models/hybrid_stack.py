"""Device weights of hybrid recurrent / windowed-attention stacks (the Tudilix design) in the forms the kernels consume.

Everything that reads the same row is one matrix (`w_in`): queries, keys and values of an attention layer, or the two branches of a
recurrent one.  The two block-diagonal gates of a recurrence are one product grouped over the blocks (`w_gates`, per block the decay
gate's rows, then the input gate's).  Norm weights (stored as distances from one) become plain gains, lambda becomes the log decay at an open gate.

Widths are padded so that every operand row starts on a 16-byte boundary (multiples of 8); pads are zero in the weights, so they stay
zero in the activations.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .. import ops
from ..config import AttentionSpec, ModelSpec, RecurrentSpec
from ..ops import KIND_BF16, KIND_F32, TcWeight
from .latent_stack import _pad, stack_kind, up
from .weights import DeviceWeights, LayerWeights

DECAY_SHARPNESS = 8.0


@dataclass
class HybridLayer(LayerWeights):
    """`attn_norm` / `ffn_norm` are the gains in front of the sub-layers; the feed-forward uses `ws_gate`, `ws_up`, `ws_down`."""
    attn_post: torch.Tensor | None = None       # gains of the norms behind the sub-layers
    ffn_post: torch.Tensor | None = None
    w_in: TcWeight | None = None                # [queries | keys | values] or [y branch | x branch], each branch padded to 8 rows
    conv: torch.Tensor | None = None            # [taps, channels] fp32; attention: the channels of `w_in` in order
    # recurrence
    conv_b: torch.Tensor | None = None
    y_b: torch.Tensor | None = None
    x_b: torch.Tensor | None = None
    w_gates: TcWeight | None = None             # G = blocks, [2 n, n_pad]
    gates_b: torch.Tensor | None = None         # [blocks * 2 n], the order of the product's columns
    decay: torch.Tensor | None = None           # [width]: -8 softplus(lambda)
    # feed-forward biases
    gate_b: torch.Tensor | None = None
    up_b: torch.Tensor | None = None
    down_b: torch.Tensor | None = None


@dataclass
class HybridWeights(DeviceWeights):
    rope: dict | None = None                    # rotation -> (frequencies fp32 [2, pairs]: value and rounding error, factor on cos and sin)

    @property
    def f32(self) -> bool:
        return self.lm_head.kind == KIND_F32


def rope_key(a: AttentionSpec | RecurrentSpec) -> tuple:
    return (a.rope_dims, a.rope_theta, getattr(a, "rope_scaling", None), getattr(a, "rope_divisor", 1.0))


def rope_frequencies(a: AttentionSpec | RecurrentSpec) -> tuple[list, float]:
    """Angle per position of every rotated pair, and the factor on cosine and sine."""
    n, s = a.rope_dims, getattr(a, "rope_scaling", None)
    freq = [a.rope_theta ** (-2.0 * i / n) / getattr(a, "rope_divisor", 1.0) for i in range(n // 2)]
    if s is None:
        return freq, 1.0
    edge = lambda turns: n * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(a.rope_theta))
    lo, hi = max(math.floor(edge(s.fast)), 0), min(math.ceil(edge(s.slow)), n - 1)
    ramp = [min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001))) for i in range(n // 2)]
    return [f * (1.0 - r) + f / s.factor * r for f, r in zip(freq, ramp)], 0.1 * math.log(s.factor) + 1.0


def rope_tables(spec: ModelSpec, device) -> dict:
    out = {}
    for m in [m for b in spec.blocks for m in (b.attn, b.rec) if m is not None]:
        if not m.rope_dims or rope_key(m) in out:
            continue
        freq, amp = rope_frequencies(m)
        f = torch.tensor(freq, dtype=torch.float64)
        hi = f.float()
        out[rope_key(m)] = (torch.stack([hi, (f - hi.double()).float()]).to(device).contiguous(), amp)
    return out


def hybrid_weights_from_masters(spec: ModelSpec, masters: dict, device) -> HybridWeights:
    """`masters` as `loader.stack_checkpoint.read_hybrid_masters` returns them (any floating dtype)."""
    kind = stack_kind(spec)
    W, Wp = spec.hidden, up(spec.hidden, 8)
    vec = lambda t, n: _pad(t.float().reshape(-1), n).to(device).contiguous()
    gain = lambda t: vec(1.0 + t.float(), Wp)
    mat = lambda t, *shape: TcWeight.from_master(_pad(t, *shape), kind, device)
    taps_first = lambda t: t.float().T.to(device).contiguous()

    def layer(b, lw) -> HybridLayer:
        out = HybridLayer(attn_norm=gain(lw["norm1"]), ffn_norm=None, wqkv=None, wo=None, attn_post=gain(lw["norm1b"]))
        if b.rec is not None:
            n, nb = b.rec.width, b.rec.blocks
            sq, n8 = n // nb, up(n, 8)
            out.w_in = mat(torch.cat([_pad(lw["wy"], n8, W), _pad(lw["wx"], n8, W)]), 2 * n8, Wp)
            out.y_b, out.x_b, out.conv, out.conv_b = vec(lw["y_b"], n), vec(lw["x_b"], n), taps_first(lw["conv"]), vec(lw["conv_b"], n)
            out.w_gates = mat(torch.cat([lw["ra"], lw["ri"]], 1), nb, 2 * sq, up(sq, 8))
            out.gates_b = vec(torch.cat([lw["ra_b"].reshape(nb, sq), lw["ri_b"].reshape(nb, sq)], 1), 2 * n)
            out.decay = vec(-DECAY_SHARPNESS * F.softplus(lw["lam"].double()), n)
            out.wo = mat(lw["wo"], Wp, n8)
        else:
            own = ("q", "k", "v") if b.attn.kv_from < 0 else ("q",)
            w = torch.cat([lw[f"w{k}"] for k in own])
            out.w_in, out.conv = mat(w, w.shape[0], Wp), taps_first(torch.cat([lw[f"{k}_conv"] for k in own]))
            out.q_norm = vec(lw["q_norm"], b.attn.head_dim)
            out.k_norm = vec(lw["k_norm"], b.attn.head_dim) if "k" in own else None
            out.wo = mat(lw["wo"], Wp, up(b.attn.n_heads * b.attn.v_head_dim, 8))
        if b.ffn is not None:
            f8 = up(b.ffn.intermediate, 8)
            out.ffn_norm, out.ffn_post = gain(lw["norm2"]), gain(lw["norm2b"])
            out.ws_gate, out.ws_up, out.ws_down = mat(lw["w_gate"], f8, Wp), mat(lw["w_up"], f8, Wp), mat(lw["w_down"], Wp, f8)
            out.gate_b, out.up_b, out.down_b = vec(lw["gate_b"], f8), vec(lw["up_b"], f8), vec(lw["down_b"], Wp)
        return out

    hw = HybridWeights(spec=spec, embed=_pad(masters["embed"].to(torch.bfloat16), spec.vocab, Wp).to(device).contiguous(), final_norm=gain(masters["final_norm"]),
                       lm_head=mat(masters["lm_head"], spec.vocab, Wp), rope=rope_tables(spec, device))
    hw.layers = [layer(b, lw) for b, lw in zip(spec.blocks, masters["layers"])]
    hw.layer_map = list(range(spec.n_layers))
    return hw


def hybrid_weights_random(spec: ModelSpec, device, seed: int = 1) -> HybridWeights:
    """Random weights directly on the device (benchmarks of real layer sizes)."""
    kind = stack_kind(spec)
    W = spec.hidden
    if W % 8:
        raise ValueError("random weights: the residual width must be a multiple of 8")
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

    def layer(b) -> HybridLayer:
        out = HybridLayer(attn_norm=ones(W), ffn_norm=None, wqkv=None, wo=None, attn_post=ones(W))
        if b.rec is not None:
            n, nb = b.rec.width, b.rec.blocks
            sq, n8 = n // nb, up(n, 8)
            if n % 8:
                raise ValueError("random weights: recurrent widths must be multiples of 8")
            out.w_in, out.wo = R(1, 2 * n8, W), R(1, W, n8)
            out.y_b, out.x_b, out.conv, out.conv_b = nrm(n, std=0.1), nrm(n, std=0.1), nrm(b.rec.conv_taps, n, std=0.5), nrm(n, std=0.1)
            out.w_gates, out.gates_b = R(nb, 2 * sq, up(sq, 8), keep=(2 * sq, sq)), nrm(2 * n, std=1.0)
            out.decay = -DECAY_SHARPNESS * F.softplus(nrm(n, std=1.0) - 4.0)
        else:
            a = b.attn
            dv, C = a.n_heads * a.v_head_dim, a.n_heads * a.head_dim + a.kv_token_elems
            out.w_in, out.conv, out.wo = R(1, C, W), nrm(a.conv_taps, C, std=0.5), R(1, W, up(dv, 8), keep=(W, dv))
            out.q_norm, out.k_norm = ones(a.head_dim), ones(a.head_dim) if a.kv_from < 0 else None
        if b.ffn is not None:
            ff, f8 = b.ffn.intermediate, up(b.ffn.intermediate, 8)
            out.ffn_norm, out.ffn_post = ones(W), ones(W)
            out.ws_gate, out.ws_up, out.ws_down = R(1, f8, W, keep=(ff, W)), R(1, f8, W, keep=(ff, W)), R(1, W, f8, keep=(W, ff))
            out.gate_b, out.up_b, out.down_b = torch.zeros(f8, device=device), torch.zeros(f8, device=device), nrm(W, std=0.1)
        return out

    hw = HybridWeights(spec=spec, embed=nrm(spec.vocab, W, std=1.0).to(torch.bfloat16), final_norm=ones(W), lm_head=R(1, spec.vocab, W), rope=rope_tables(spec, device))
    hw.layers = [layer(b) for b in spec.blocks]
    hw.layer_map = list(range(spec.n_layers))
    return hw

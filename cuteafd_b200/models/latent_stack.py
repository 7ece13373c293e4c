"""Device weights of latent-attention layer stacks (the Bedovik design) in the forms the kernels consume.

Everything that reads the same row is one matrix: a layer's queries, latent, head gates and router logits come from ONE product with the
stacked weight `w_in` (fp32 output, so the norm, the gates and the router see unrounded values).  The key and value expansions are kept
per head in absorbed form (`w_uk_t` folds keys into the query, `w_uv` is applied to the attended latent) and, on first use, stacked as
`w_kvb` for prefill chunks, which expand the context once per chunk.

Widths are padded so that every operand row starts on a 16-byte boundary (residual width and feed-forward width to 8, latents and
per-head query widths to whole 64-element chunks); pads are zero in the weights, so they stay zero in the activations.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..config import AttentionSpec, ModelSpec
from ..ops import KIND_BF16, KIND_F32, TcWeight
from .weights import DeviceWeights, LayerWeights


def up(n: int, m: int) -> int:
    return -(-n // m) * m


@dataclass
class StackLayer(LayerWeights):
    """`attn_norm` is the Dynamic Tanh gain; `wo`, `w_up` and `w_down` (the experts) keep their usual fields, `w_gate` stays None."""
    norm_b: torch.Tensor | None = None
    norm_alpha: float = 1.0
    w_in: TcWeight | None = None            # rows: H * dim queries | rank latent | H gates (if any) | experts' router logits
    kv_norm: torch.Tensor | None = None
    w_uk_t: TcWeight | None = None          # G = H, [rank_pad, dim_pad]
    w_uv: TcWeight | None = None            # G = H, [vdim, rank_pad]
    w_kvb: TcWeight | None = None           # [H * (dim_pad + vdim_pad), rank_pad], prefill only
    ls1: torch.Tensor | None = None
    ls2: torch.Tensor | None = None

    @property
    def norm(self) -> tuple:
        return self.attn_norm, self.norm_b, self.norm_alpha

    def ensure_kvb(self) -> TcWeight:
        """Per head: the key rows (padded to dim_pad), then the value rows (padded to whole 64-row chunks)."""
        if self.w_kvb is None:
            uk, uv = self.w_uk_t.data, self.w_uv.data                  # [H, rank_pad, dim_pad], [H, vdim, rank_pad]
            H, rp, dp = uk.shape
            dvp = up(uv.shape[1], 64)
            data = torch.zeros(H, dp + dvp, rp, dtype=uk.dtype, device=uk.device)
            data[:, :dp] = uk.transpose(1, 2)
            data[:, dp:dp + uv.shape[1]] = uv
            data = data.reshape(1, H * (dp + dvp), rp)
            self.w_kvb = TcWeight(KIND_BF16, 1, data.shape[1], rp, data, ops.encode_tmap(data, 128))
        return self.w_kvb


@dataclass
class StackWeights(DeviceWeights):
    """`embed` and `pos` stay bf16 tables in either mode (they are read, not multiplied)."""
    pos: torch.Tensor | None = None
    final_b: torch.Tensor | None = None
    final_alpha: float = 1.0
    loop_in: TcWeight | None = None         # [hidden_pad, 2 * hidden_pad]: [x | embedding output]
    loop_step: torch.Tensor | None = None   # [times, hidden_pad] fp32

    @property
    def f32(self) -> bool:
        return self.lm_head.kind == KIND_F32

    def nbytes(self) -> int:
        return super().nbytes() + (self.pos.numel() * 2 if self.pos is not None else 0) + (self.loop_in.nbytes if self.loop_in is not None else 0)


def _pad(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """Zero-pads `t` to `shape` (leading corner kept)."""
    if tuple(t.shape) == shape:
        return t
    out = t.new_zeros(shape)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


def stack_kind(spec: ModelSpec) -> str:
    if spec.quant.dense not in ("bf16", "f32") or spec.quant.experts != spec.quant.dense:
        raise ValueError("layer stacks run with bf16 or fp32 weights (dense and experts alike)")
    return spec.quant.dense


def stack_weights_from_masters(spec: ModelSpec, masters: dict, device) -> StackWeights:
    """`masters`: "embed", "pos", "lm_head", "final_norm" = (w, b, alpha), with a loop "loop_in" and "loop_step", and per layer "norm" =
    (w, b, alpha), "wq", "w_dkv", "kv_norm", "w_uk", "w_uv", "wo", "ls1" and, where the layer has them, "w_g", "ls2", "router", "w_up",
    "w_down" - matrices [out, in] (experts stacked), any floating dtype."""
    kind = stack_kind(spec)
    W = spec.hidden
    Wp = up(W, 8)
    vec = lambda t, n: _pad(t.float().reshape(-1), n).to(device).contiguous()
    mat = lambda t, *shape: TcWeight.from_master(_pad(t, *shape), kind, device)

    def layer(b, lw) -> StackLayer:
        a, m = b.attn, b.moe
        H, d, dv, r = a.n_heads, a.head_dim, a.v_head_dim, a.kv_lora_rank
        rp, dp = up(r, 64), up(d, 64)
        rows = [lw["wq"], lw["w_dkv"]] + ([lw["w_g"]] if a.out_gate else []) + ([lw["router"]] if m is not None else [])
        w_in = torch.cat([t.float() if kind == "f32" else t.to(torch.bfloat16) for t in rows], 0)
        uk_t = _pad(lw["w_uk"].reshape(H, d, r).transpose(1, 2), H, rp, dp)
        nw, nb, al = lw["norm"]
        out = StackLayer(attn_norm=vec(nw, Wp), ffn_norm=None, wqkv=None, wo=mat(lw["wo"], Wp, up(H * dv, 8)), norm_b=vec(nb, Wp), norm_alpha=float(al),
                         w_in=mat(w_in, w_in.shape[0], Wp), kv_norm=vec(lw["kv_norm"], r), w_uk_t=TcWeight.from_master(uk_t, kind, device),
                         w_uv=mat(lw["w_uv"].reshape(H, dv, r), H, dv, rp), ls1=vec(lw["ls1"], Wp))
        if m is not None:
            E, ff = m.n_experts, m.intermediate
            out.w_up, out.w_down = mat(lw["w_up"], E, ff, Wp), mat(lw["w_down"], E, Wp, up(ff, 8))
            out.ls2 = vec(lw["ls2"], Wp)
        return out

    table = lambda t: _pad(t.to(torch.bfloat16), t.shape[0], Wp).to(device).contiguous()
    fw, fb, fa = masters["final_norm"]
    sw = StackWeights(spec=spec, embed=table(masters["embed"]), final_norm=vec(fw, Wp), lm_head=mat(masters["lm_head"], spec.vocab, Wp),
                      pos=table(masters["pos"]) if spec.learned_positions else None, final_b=vec(fb, Wp), final_alpha=float(fa))
    if spec.loop is not None:
        wi = masters["loop_in"]
        sw.loop_in = mat(torch.cat([_pad(wi[:, :W], Wp, Wp), _pad(wi[:, W:], Wp, Wp)], 1), Wp, 2 * Wp)
        sw.loop_step = _pad(masters["loop_step"].float(), spec.loop.times, Wp).to(device).contiguous()
    sw.layers = [layer(b, lw) for b, lw in zip(spec.blocks, masters["layers"])]
    sw.layer_map = list(range(spec.n_layers))
    return sw


def stack_weights_random(spec: ModelSpec, device, seed: int = 1) -> StackWeights:
    """Random weights directly on the device (benchmarks of real layer sizes)."""
    kind = stack_kind(spec)
    W = spec.hidden
    if W % 8:
        raise ValueError("random weights: the residual width must be a multiple of 8")
    gen = torch.Generator(device=device).manual_seed(seed)
    nrm = lambda *s, std: torch.empty(*s, device=device).normal_(0, std, generator=gen)
    ones = lambda n: torch.ones(n, dtype=torch.float32, device=device)
    zeros = lambda n: torch.zeros(n, dtype=torch.float32, device=device)

    def R(G, N, K, std=None, keep=None):
        """Random [G, N, K] whose pads beyond `keep` = (rows, columns) are zero."""
        data = torch.empty(G, N, K, dtype=torch.bfloat16 if kind == "bf16" else torch.float32, device=device).normal_(0, std or K ** -0.5, generator=gen)
        if keep:
            data[:, keep[0]:] = 0
            data[:, :, keep[1]:] = 0
        return TcWeight(KIND_BF16, G, N, K, data, ops.encode_tmap(data, 128)) if kind == "bf16" else TcWeight(KIND_F32, G, N, K, data, None)

    def layer(b) -> StackLayer:
        a, m = b.attn, b.moe
        H, d, dv, r = a.n_heads, a.head_dim, a.v_head_dim, a.kv_lora_rank
        rp, dp = up(r, 64), up(d, 64)
        out = StackLayer(attn_norm=ones(W), ffn_norm=None, wqkv=None, wo=R(1, W, up(H * dv, 8), keep=(W, H * dv)), norm_b=zeros(W), norm_alpha=0.7,
                         w_in=R(1, H * d + r + (H if a.out_gate else 0) + (m.n_experts if m else 0), W), kv_norm=ones(r),
                         w_uk_t=R(H, rp, dp, std=r ** -0.5, keep=(r, d)), w_uv=R(H, dv, rp, std=r ** -0.5, keep=(dv, r)), ls1=ones(W) * 0.5)
        if m is not None:
            out.w_up, out.w_down = R(m.n_experts, m.intermediate, W), R(m.n_experts, W, up(m.intermediate, 8), keep=(W, m.intermediate))
            out.ls2 = ones(W) * 0.5
        return out

    sw = StackWeights(spec=spec, embed=nrm(spec.vocab, W, std=1.0).to(torch.bfloat16), final_norm=ones(W), lm_head=R(1, spec.vocab, W),
                      pos=nrm(spec.learned_positions, W, std=0.1).to(torch.bfloat16) if spec.learned_positions else None, final_b=zeros(W), final_alpha=0.7)
    if spec.loop is not None:
        sw.loop_in, sw.loop_step = R(1, W, 2 * W), nrm(spec.loop.times, W, std=0.1)
    sw.layers = [layer(b) for b in spec.blocks]
    sw.layer_map = list(range(spec.n_layers))
    return sw

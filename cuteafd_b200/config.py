"""Model geometry and deployment descriptions.

A `ModelSpec` is the single description every layer of the framework consumes: the
CPU oracle, the weight initialiser, the planner/placement solver, the engine and the
benchmarks.  The reference derives the same facts from a snapshot's `config.json`
(reference: rust/crates/cuteafd-loader/src/plan/family.rs, cuteafd-core/src/constants.rs);
here they are plain dataclasses plus a `from_hf_config` reader.
"""
from __future__ import annotations

import dataclasses
import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import Optional


@dataclass(frozen=True)
class AttentionSpec:
    # "gqa" | "mla" | per layer of a stack (BlockSpec): "latent" (latent attention without positions), "conv_gqa" (grouped-query attention
    # whose projections pass a short causal convolution)
    kind: str = "gqa"
    n_heads: int = 8
    n_kv_heads: int = 2
    head_dim: int = 32
    rope_theta: float = 10000.0
    rope_interleaved: bool = True   # pair (2i, 2i+1) rotation; False = half-split (HF llama style)
    qk_norm: bool = False           # per-head RMSNorm on q and k (Qwen3)
    # MLA (DeepSeek-V3 style); ignored for gqa
    q_lora_rank: int = 0
    kv_lora_rank: int = 0
    qk_nope_head_dim: int = 0
    qk_rope_head_dim: int = 0
    v_head_dim: int = 0
    window: int = 0                 # sliding window (0 = full)
    sink: bool = False              # learned attention sink logit per head
    # Hybrid stacks (MiMo-V2 style: full causal layers interleaved with sliding-window layers that carry the sinks): with
    # full_every = n > 0, layers i with i % n == 0 are full attention (no window, no sink, `rope_theta`), the others use `window`,
    # the sink and `swa_rope_theta` (0 = the same theta).  0 = every layer as configured above.
    full_every: int = 0
    swa_rope_theta: float = 0.0
    # Sparse attention with a learned indexer (DSA of the DeepSeek-V3.2 / GLM-5 lines; MLA only): with index_topk = k > 0 every
    # query token scores the visible cached positions with `index_heads` small heads of `index_dim` dimensions
    # (score = sum_h w_h * relu(q_h . k)), and attends only to its k best positions once it can see more than k.
    index_topk: int = 0
    index_heads: int = 32
    index_dim: int = 128
    # Hybrid stacks with linear-attention layers (the Qwen 3.8 / GLM 5.3 Flash lines; GQA models only): with linear_every = n > 0,
    # layer i is a full-attention layer when (i + 1) % n == 0 and a gated delta-rule layer otherwise (n = 4: three linear layers,
    # then one full).  Linear layers have `linear_k_heads` query / key heads and `linear_v_heads` value heads of 128 dimensions,
    # a width-4 causal convolution in front of q / k / v, and a per-sequence recurrent state instead of KV pages.
    # `linear_per_channel`: one decay per key channel (KDA) instead of one per head (GDN).
    linear_every: int = 0
    linear_k_heads: int = 2
    linear_v_heads: int = 4
    linear_per_channel: bool = False
    # Latent attention without a rotated part (kind "latent"): head_dim, v_head_dim and kv_lora_rank as above, `scale` multiplies the scores
    # (0 = head_dim ** -0.5), `out_gate` multiplies each head's output by a sigmoid of the layer's input.
    scale: float = 0.0
    out_gate: bool = False
    # Kind "conv_gqa": head_dim, v_head_dim, window, qk_norm and scale as above, `conv_taps` of the convolution on q, k and v, the first
    # `rope_dims` dimensions of a head rotated (interleaved pairs, `rope_theta`, `rope_scaling`), and with kv_from >= 0 the keys and values
    # of that layer instead of own ones.
    conv_taps: int = 1
    rope_dims: int = 0
    rope_scaling: Optional["RopeScaling"] = None
    kv_from: int = -1
    # Kind "conv_gqa" in hyper-connected stacks, besides: no convolution with `conv_taps` 0; `keep_first` keys of the sequence stay visible behind the window; `sink`; one norm over
    # all heads of q (and of k) at once; keys that are also the values (as they leave the convolution, no value projection); biases of the
    # projections; an output gate with one number per head (`out_gate`) or, with `gate_values`, one per output value.
    keep_first: int = 0
    qk_norm_whole: bool = False
    values_are_keys: bool = False
    qkv_bias: bool = False
    out_bias: bool = False
    gate_values: bool = False
    # Kind "conv_gqa" in mixed stacks, besides: one key and value for each block of `pool` tokens that lies wholly in front of the window (the means of
    # the tokens' cached keys and values); queries and keys over their root mean square per head, without gains; every angle of the rotation divided by
    # `rope_divisor`.
    # Kind "latent" in mixed stacks, besides: queries through a latent of their own (`q_lora_rank` > 0), a rotated part of `rope_dims` dimensions behind
    # the `head_dim` unrotated ones (one rotated key part shared by the heads, cached beside the latent), `sink`.
    pool: int = 0
    qk_norm_unit: bool = False
    rope_divisor: float = 1.0

    @property
    def latent_row(self) -> int:
        """Elements of a cached row of kind "latent": latent and rotated key part in whole 64-element chunks."""
        return -(-self.kv_lora_rank // 64) * 64 + -(-self.rope_dims // 64) * 64

    @property
    def pooled_page_rows(self) -> int:
        """Rows of pooled blocks that belong to a page of 64 tokens: whole strips of eight blocks, each with the page of its first token."""
        return 8 * -(-8 // self.pool) if self.pool else 0

    @property
    def gate_width(self) -> int:
        """Numbers of the output gate per token."""
        return 0 if not self.out_gate else (self.n_heads * self.v_head_dim if self.gate_values else self.n_heads)

    @property
    def conv_channels(self) -> int:
        """Projected channels in front of the convolution (kind "conv_gqa")."""
        return self.n_heads * self.head_dim + (self.kv_token_elems if not self.values_are_keys else self.n_kv_heads * self.head_dim)

    @property
    def softmax_scale(self) -> float:
        return self.scale or self.head_dim ** -0.5

    @property
    def q_dim(self) -> int:
        if self.kind == "mla":
            return self.n_heads * (self.qk_nope_head_dim + self.qk_rope_head_dim)
        return self.n_heads * self.head_dim

    @property
    def kv_token_elems(self) -> int:
        """Cached elements per token per layer."""
        if self.kind == "mla":
            return self.kv_lora_rank + self.qk_rope_head_dim
        if self.kind == "latent":
            return self.kv_lora_rank + self.rope_dims
        if self.kind == "conv_gqa":
            return 0 if self.kv_from >= 0 else self.n_kv_heads * (self.head_dim + self.v_head_dim)
        return 2 * self.n_kv_heads * self.head_dim


@dataclass(frozen=True)
class RopeScaling:
    """YaRN: frequencies that turn fewer than `slow` times over `original` positions are divided by `factor`, those that turn more than
    `fast` times stay, with a linear ramp over the pairs between; cosine and sine grow by 0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class MoESpec:
    n_experts: int = 16
    top_k: int = 4
    intermediate: int = 128
    n_shared: int = 1
    shared_intermediate: int = 0    # 0 -> n_shared * intermediate
    scoring: str = "sigmoid"        # sigmoid | softmax | sqrtsoftplus | hash
    normalize: bool = True
    route_scale: float = 1.0
    use_bias: bool = False          # noaux_tc selection bias (affects choice only)
    n_group: int = 1
    topk_group: int = 1
    first_dense: int = 0            # leading dense layers
    dense_intermediate: int = 0
    swiglu_limit: float = 0.0       # clamp on gate/up (0 = off)
    activation: str = "swiglu"      # "swiglu" (gate and up projections) | "relu2" (up projection only, squared ReLU)
    group_score: str = "top2"       # what ranks a group of experts: the sum of its two best scores, or its best one ("max")

    @property
    def shared_inter(self) -> int:
        return self.shared_intermediate or self.n_shared * self.intermediate


@dataclass(frozen=True)
class QuantSpec:
    """Weight formats as shipped in the checkpoint (no repacking on disk)."""
    experts: str = "bf16"           # bf16 | fp8_block128 | mxfp4 | nvfp4 | exl3
    dense: str = "bf16"             # bf16 | fp8_block128 | fp8_block32 | nvfp4
    kv: str = "bf16"                # bf16 | fp8
    exl3_bits: int = 4


@dataclass(frozen=True)
class RecurrentSpec:
    """A recurrent mixer.  "rglru": two branches of `width` channels, one gated by GELU, the other through a convolution of `conv_taps` and a
    real-gated linear recurrence whose two gates are block-diagonal (`blocks` square blocks).
    Linear attention of `heads` heads with a state of `dim` x `vdim` each: "retention" (a constant decay per head, `decay`; the first `rope_dims`
    dimensions of q and k rotated, i with i + rope_dims / 2) and "gla" (a decay per key channel and token, the sigmoid of a projection of rank
    `rank` to the power 1 / `tau`; rank 0: as wide as the snapshot's tensors).  "hgrn2" writes with what its forget gate gives up: a gate per channel
    between a learned lower bound and one is the decay, one minus it the key; SiLU on q, an output norm, no output gate."""
    kind: str = "rglru"
    width: int = 256
    blocks: int = 1
    conv_taps: int = 4
    heads: int = 0
    dim: int = 0
    vdim: int = 0
    decay: tuple = ()
    rope_dims: int = 0
    rope_theta: float = 10000.0
    tau: float = 1.0
    rank: int = 0


@dataclass(frozen=True)
class DenseFfnSpec:
    """A dense feed-forward.  "clamped_glu": gate g = min(., limit), linear half u clamped to [-limit, limit], g sigmoid(1.702 g) (u + 1);
    biases on all three projections.  "silu_glu": silu(g) u, no biases."""
    intermediate: int
    limit: float = 0.0
    activation: str = "clamped_glu"


@dataclass(frozen=True)
class BlockSpec:
    """One layer of a stack whose layers differ: its mixer (attention, or a recurrent one) and its feed-forward (routed experts, dense, or
    neither: the layer has none).  A layer with both mixers runs them side by side on the same input and adds their outputs, `merge_scales`
    times each, with `merge_norm` behind an RMS norm each."""
    attn: Optional[AttentionSpec] = field(default_factory=lambda: AttentionSpec(kind="latent"))
    moe: Optional[MoESpec] = None
    rec: Optional[RecurrentSpec] = None
    ffn: Optional[DenseFfnSpec] = None
    merge_scales: tuple = (1.0, 1.0)
    merge_norm: bool = False


@dataclass(frozen=True)
class PairTableSpec:
    """A table added to the token embedding, addressed by the token and the one before it: row (previous * mul_prev + token * mul_cur) mod buckets;
    the row behind the last starts a sequence."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LoopSpec:
    """Layers [start, stop) run `times` times in a row with the same weights and a cache (and state) of their own per pass.  With entry "project" each
    pass opens with a projection of [x; embedding output] and a learned vector of the pass; with "add" every pass but the first opens by adding the
    embedding output to x."""
    start: int
    stop: int
    times: int
    entry: str = "project"


@dataclass(frozen=True)
class ModelSpec:
    name: str = "tiny"
    family: str = "tiny"
    vocab: int = 1024
    hidden: int = 256
    n_layers: int = 2
    rms_eps: float = 1e-5
    attn: AttentionSpec = field(default_factory=AttentionSpec)
    moe: MoESpec = field(default_factory=MoESpec)
    quant: QuantSpec = field(default_factory=QuantSpec)
    mtp_layers: int = 0             # native next-n (MTP) draft layers
    # Hyper-connections (the V4 line): 0 = one residual stream; 4 = four streams mixed at every sub-layer boundary by per-token
    # coefficients (collapse weights, spread weights and a Sinkhorn-normalised 4 x 4 stream mix from 24 projections of the row)
    hyper_streams: int = 0
    hyper_sinkhorn_iters: int = 20
    # N-gram memory (the V4.1 line's "engram"): decoder layers whose input takes a gated projection of hashed table rows addressed by the
    # 2- to 4-grams ending at the token; the tables have engram_prime_floor-sized heads (24 consecutive primes above it per layer)
    engram_layers: tuple = ()
    engram_row_dim: int = 256
    engram_prime_floor: int = 500
    engram_vocab: int = 0           # compressed vocabulary of the addressing (0: the model's vocabulary, identity map)
    init_std: float = 0.02
    tie_embeddings: bool = False
    max_context: int = 1 << 20
    # Stacks of unequal layers (`blocks` non-empty; `attn` / `moe` above then describe the first layer of their kind), over an fp32 residual.
    # "latent" stacks: parallel layers (one norm, attention and feed-forward read it, both scaled per channel and added), Dynamic Tanh for a
    # norm.  "hybrid" stacks: windowed attention and recurrent layers, RMS norms in front of and behind every sub-layer, whose result is
    # added `residual_mult` times; logits bounded by `logit_softcap` (0 = not).  "hyper" stacks (`streams` > 0): that many residual streams with
    # constant weights per sub-layer (how it reads them, how its output and the old streams make the new ones); mixers alone or side by side.
    # "mixed" stacks (`mixed`): parallel layers of attention with pooled blocks, rotated latent attention and HGRN2; mixer and feed-forward read the same
    # RMS-normed row, each times a number of its own; behind a layer the token's part of a second table (`side_dim` values per layer, gated by the
    # residual) is projected, normalised and added; the embedding is multiplied by `embed_scale`.
    blocks: tuple = ()
    mixed: bool = False
    embed_scale: float = 1.0
    side_dim: int = 0
    streams: int = 0
    pair_table: Optional[PairTableSpec] = None
    residual_mult: float = 1.0
    logit_softcap: float = 0.0
    loop: Optional[LoopSpec] = None
    learned_positions: int = 0      # rows of the learned position table (0 = none); also the longest context

    @property
    def stack(self) -> str:
        """Which kind of stack `blocks` describes: "latent", "hybrid", "hyper", "mixed", or "" for models without blocks."""
        if not self.blocks:
            return ""
        if self.mixed:
            return "mixed"
        if self.streams:
            return "hyper"
        return "latent" if all(b.attn is not None and b.attn.kind == "latent" for b in self.blocks) else "hybrid"

    def kv_layers(self) -> list:
        """Layers of a hybrid or hyper-connected stack that keep keys and values of their own."""
        return [i for i, b in enumerate(self.blocks) if b.attn is not None and b.attn.kv_from < 0]

    def layer_runs(self) -> list:
        """[(layer, pass index where a pass of the loop opens with this run, else None)] in the order the layers run."""
        lp, n = self.loop, self.n_layers
        if lp is None:
            return [(i, None) for i in range(n)]
        return ([(i, None) for i in range(lp.start)] + [(i, t if i == lp.start else None) for t in range(lp.times) for i in range(lp.start, lp.stop)] +
                [(i, None) for i in range(lp.stop, n)])

    def attention_runs(self, kind: str) -> list:
        """Layer runs (their numbers in `layer_runs`) whose mixer is attention of this kind: each keeps a cache plane of its own in a mixed stack."""
        return [r for r, (i, _) in enumerate(self.layer_runs()) if self.blocks[i].attn is not None and self.blocks[i].attn.kind == kind]

    def replace(self, **kw) -> "ModelSpec":
        return dataclasses.replace(self, **kw)

    def engram_spec(self):
        """Addressing / shape of the n-gram memory, or None for models without one."""
        if not self.engram_layers:
            return None
        from .ref.engram import EngramSpec
        return EngramSpec(layers=tuple(self.engram_layers), vocab=self.engram_vocab or self.vocab, pad_id=0, row_dim=self.engram_row_dim,
                          prime_floor=self.engram_prime_floor, streams=1, hidden=self.hidden)

    # ---- per-layer attention program ---------------------------------------
    def layer_is_full(self, layer: int) -> bool:
        """Full causal attention (True) or the sliding-window variant (False); MTP draft layers (>= n_layers) are full."""
        a = self.attn
        if a.full_every <= 0:
            return a.window == 0
        return layer >= self.n_layers or layer % a.full_every == 0

    def layer_is_linear(self, layer: int) -> bool:
        """A gated delta-rule (linear attention) layer; MTP draft layers (>= n_layers) are full-attention layers."""
        n = self.attn.linear_every
        return n > 0 and layer < self.n_layers and (layer + 1) % n != 0

    def layer_window(self, layer: int) -> int:
        a = self.attn
        return a.window if (a.full_every <= 0 or not self.layer_is_full(layer)) else 0

    def layer_has_sink(self, layer: int) -> bool:
        a = self.attn
        return a.sink and (a.full_every <= 0 or not self.layer_is_full(layer))

    def layer_rope_theta(self, layer: int) -> float:
        a = self.attn
        if a.full_every > 0 and a.swa_rope_theta and not self.layer_is_full(layer):
            return a.swa_rope_theta
        return a.rope_theta

    # ---- derived sizes -------------------------------------------------
    def is_moe_layer(self, layer: int) -> bool:
        return layer >= self.moe.first_dense

    def expert_params(self) -> int:
        return 3 * self.hidden * self.moe.intermediate

    def attn_params(self, attn: Optional[AttentionSpec] = None) -> int:
        a, h = attn or self.attn, self.hidden
        if a.kind == "conv_gqa":
            return h * (a.conv_channels + a.gate_width + a.n_heads * a.v_head_dim)
        if a.kind == "latent":
            qd = a.n_heads * (a.head_dim + a.rope_dims)
            return ((h * a.q_lora_rank + a.q_lora_rank * qd if a.q_lora_rank else h * qd) + h * (a.kv_lora_rank + a.rope_dims + (a.n_heads if a.out_gate else 0)) +
                    a.n_heads * (a.head_dim + a.v_head_dim) * a.kv_lora_rank + a.n_heads * a.v_head_dim * h)
        if a.kind == "mla":
            qk = a.qk_nope_head_dim + a.qk_rope_head_dim
            q = h * a.q_lora_rank + a.q_lora_rank * a.n_heads * qk if a.q_lora_rank else h * a.n_heads * qk
            kv = h * (a.kv_lora_rank + a.qk_rope_head_dim) + a.kv_lora_rank * a.n_heads * (a.qk_nope_head_dim + a.v_head_dim)
            return q + kv + a.n_heads * a.v_head_dim * h
        return h * (a.n_heads + 2 * a.n_kv_heads) * a.head_dim + a.n_heads * a.head_dim * h

    def bits(self, fmt: str) -> float:
        return {"f32": 32.0, "bf16": 16.0, "fp8_block128": 8.0 + 32.0 / (128 * 128), "fp8_block32": 8.0 + 8.0 / (32 * 32),
                "mxfp4": 4.25, "nvfp4": 4.5, "exl3": float(self.quant.exl3_bits)}[fmt]

    def weight_bytes(self) -> dict:
        """Bytes per category for the whole model (planner input)."""
        if self.stack in ("hybrid", "hyper", "mixed"):
            db, eb, moes = self.bits(self.quant.dense) / 8, self.bits(self.quant.experts) / 8, [b.moe for b in self.blocks if b.moe is not None]
            rec = sum(self.recurrent_params(b.rec) for b in self.blocks if b.rec is not None)
            return {"routed_experts": sum(3 * self.hidden * m.intermediate * m.n_experts for m in moes) * eb,
                    "shared_experts": sum(3 * self.hidden * m.shared_inter for m in moes if m.n_shared) * db, "router": sum(m.n_experts for m in moes) * self.hidden * db,
                    "embed_head": self.vocab * self.hidden * (2 + db) + (2 * (self.pair_table.buckets + 1) * self.hidden if self.pair_table else 0) +
                                  self.n_layers * self.side_dim * (2 * self.vocab + 2 * self.hidden * db),
                    "dense_ffn": sum(3 * self.hidden * b.ffn.intermediate for b in self.blocks if b.ffn is not None) * db,
                    "attention": (rec + sum(self.attn_params(b.attn) for b in self.blocks if b.attn is not None)) * db}
        if self.blocks:
            eb, db = self.bits(self.quant.experts) / 8, self.bits(self.quant.dense) / 8
            ffs = [b.moe for b in self.blocks if b.moe is not None]
            return {"routed_experts": sum((2 if m.activation == "relu2" else 3) * self.hidden * m.intermediate * m.n_experts for m in ffs) * eb,
                    "shared_experts": 0.0, "dense_ffn": 0.0, "attention": sum(self.attn_params(b.attn) for b in self.blocks) * db,
                    "router": sum(m.n_experts for m in ffs) * self.hidden * db,
                    "embed_head": (2 * self.vocab + self.learned_positions) * self.hidden * 2 + (2 * self.hidden ** 2 * db if self.loop else 0)}
        moe_layers = self.n_layers - self.moe.first_dense
        eb = self.bits(self.quant.experts) / 8
        db = self.bits(self.quant.dense) / 8
        routed = moe_layers * self.moe.n_experts * self.expert_params() * eb
        shared = moe_layers * 3 * self.hidden * self.moe.shared_inter * db
        dense_ffn = self.moe.first_dense * 3 * self.hidden * self.moe.dense_intermediate * db
        attn = self.n_layers * self.attn_params() * db
        router = moe_layers * self.moe.n_experts * self.hidden * 2
        embed = self.vocab * self.hidden * 2 * (1 if self.tie_embeddings else 2)
        return {"routed_experts": routed, "shared_experts": shared, "dense_ffn": dense_ffn,
                "attention": attn, "router": router, "embed_head": embed}

    def recurrent_params(self, r: RecurrentSpec) -> int:
        if r.kind == "rglru":
            return 3 * self.hidden * r.width + 2 * r.width ** 2 // r.blocks
        if r.kind == "hgrn2":
            return 2 * self.hidden * r.heads * (r.dim + r.vdim)
        return self.hidden * r.heads * (2 * r.dim + 3 * r.vdim) + r.rank * (self.hidden + r.heads * r.dim)

    def kv_row_elems(self) -> int:
        """Elements of a cached token's row in a hybrid, hyper-connected or mixed stack: the widest layer's key heads, then its value heads."""
        up = lambda n: -(-n // 64) * 64
        return max((b.attn.n_kv_heads * (up(b.attn.head_dim) + up(b.attn.v_head_dim)) for b in self.blocks
                    if b.attn is not None and b.attn.kind == "conv_gqa" and b.attn.kv_from < 0), default=0)

    def latent_row_elems(self) -> int:
        """Elements of a cached token's latent row in a mixed stack: the widest layer's."""
        return max((b.attn.latent_row for b in self.blocks if b.attn is not None and b.attn.kind == "latent"), default=0)

    def state_bytes_per_seq(self, depth: int = 8) -> int:
        """Bytes of one sequence's state slot in a hybrid, hyper-connected or mixed stack (`engine.hybrid_stack`, `engine.hyper_stack`,
        `engine.mixed_stack`): convolution inputs and recurrent states of the last positions, `depth` of which can be taken back."""
        eb, n = 2 if self.quant.dense == "bf16" else 4, 4 * (depth + 1) if self.pair_table is not None else 0
        for b in (self.blocks[i] for i, _ in self.layer_runs()):
            r, a = b.rec, b.attn
            if r is not None and r.kind == "rglru":
                n += r.width * ((r.conv_taps - 1 + depth) * eb + (depth + 1) * 4)
            elif r is not None:         # two states, the last inputs of the recurrence, two positions per head
                vp = -(-r.vdim // 4) * 4
                n += r.heads * (4 * (2 * r.dim * vp + depth * (2 * r.dim + vp)) + 8)
            if a is not None and a.kind == "conv_gqa" and a.conv_taps:
                n += a.conv_channels * (a.conv_taps - 1 + depth) * eb
        return n

    def kv_bytes_per_token(self) -> float:
        per = {"fp8": 1.0, "f32": 4.0}.get(self.quant.kv, 2.0)
        if self.stack in ("hybrid", "hyper"):  # one row width for every layer with keys of its own, heads in whole 64-element chunks
            return len(self.kv_layers()) * self.kv_row_elems() * per
        if self.stack == "mixed":   # keys and values with their pooled blocks, and latents: a plane per layer run
            runs = [self.blocks[i].attn for i, _ in self.layer_runs()]
            pooled = sum(a.pooled_page_rows / 64 * a.n_kv_heads * (-(-a.head_dim // 64) * 64 + -(-a.v_head_dim // 64) * 64) for a in runs if a is not None and a.pool)
            return (len(self.attention_runs("conv_gqa")) * self.kv_row_elems() + len(self.attention_runs("latent")) * self.latent_row_elems() + pooled) * per
        if self.blocks:             # one row width for every layer run (the widest latent, in whole 64-element chunks)
            return len(self.layer_runs()) * max(-(-b.attn.kv_token_elems // 64) * 64 for b in self.blocks) * per
        return self.n_layers * self.attn.kv_token_elems * per


# ---------------------------------------------------------------------------
# Named configurations
# ---------------------------------------------------------------------------

def tiny_spec() -> ModelSpec:
    """Tiny synthetic MoE decoder (CPU oracle config): vocab 1024, hidden 256, 2 layers,
    GQA 8q/2kv/32, 16 experts sigmoid-normalised top-4 + 1 shared, SwiGLU I=128."""
    return ModelSpec()


def deepseek_v3_spec(n_layers: int = 61) -> ModelSpec:
    """DeepSeek-V3-shape: 61 layers, hidden 7168, MLA 128 heads (q_lora 1536, kv_lora 512,
    rope 64), 256 experts top-8 + 1 shared, I=2048, vocab 129280; FP8 128x128 dense, MXFP4 experts."""
    return ModelSpec(
        name="deepseek-v3-shape", family="deepseek_v3", vocab=129280, hidden=7168, n_layers=n_layers,
        rms_eps=1e-6,
        attn=AttentionSpec(kind="mla", n_heads=128, n_kv_heads=128, head_dim=192, rope_theta=10000.0,
                           q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128,
                           qk_rope_head_dim=64, v_head_dim=128),
        moe=MoESpec(n_experts=256, top_k=8, intermediate=2048, n_shared=1, scoring="sigmoid",
                    normalize=True, route_scale=2.5, use_bias=True, n_group=8, topk_group=4,
                    first_dense=min(3, n_layers), dense_intermediate=18432),
        quant=QuantSpec(experts="mxfp4", dense="fp8_block128", kv="bf16"),
        mtp_layers=1)


def qwen3_235b_spec(n_layers: int = 94) -> ModelSpec:
    """Qwen3-235B-A22B-shape with NVFP4 weights: 94 layers, hidden 4096, GQA 64q/4kv/128,
    128 experts top-8, I=1536, vocab 151936."""
    return ModelSpec(
        name="qwen3-235b-a22b-shape", family="qwen3_moe", vocab=151936, hidden=4096, n_layers=n_layers,
        rms_eps=1e-6,
        attn=AttentionSpec(kind="gqa", n_heads=64, n_kv_heads=4, head_dim=128, rope_theta=1e6,
                           rope_interleaved=False, qk_norm=True),
        moe=MoESpec(n_experts=128, top_k=8, intermediate=1536, n_shared=0, scoring="softmax",
                    normalize=True),
        quant=QuantSpec(experts="nvfp4", dense="nvfp4", kv="bf16"))


def ep_microbench_spec() -> ModelSpec:
    """EP dispatch -> grouped GEMM -> combine microbench layer: hidden 7168, 256 experts, top-8,
    I=2048, MXFP4 weights."""
    return ModelSpec(name="ep-microbench", family="microbench", hidden=7168, n_layers=1, vocab=1024,
                     moe=MoESpec(n_experts=256, top_k=8, intermediate=2048, n_shared=0,
                                 scoring="softmax", normalize=True),
                     quant=QuantSpec(experts="mxfp4"))


def deepseek_v32_spec(n_layers: int = 61) -> ModelSpec:
    """DeepSeek-V3.2-shape: the V3 shape with the sparse-attention indexer (64 index heads of 128, 2048 positions kept per query)."""
    base = deepseek_v3_spec(n_layers)
    return base.replace(name="deepseek-v32-shape", attn=dataclasses.replace(base.attn, index_topk=2048, index_heads=64, index_dim=128))


def hybrid_gdn_spec(n_layers: int = 48, per_channel: bool = False) -> ModelSpec:
    """Hybrid linear-attention MoE shape (the Qwen-Next line): three gated delta-rule layers (16 q/k heads, 32 value heads of 128)
    then one full GQA layer (16q/2kv/128), hidden 2048, 128 experts top-8 I=768 + 1 shared, vocab 151936, bf16 dense projections and
    NVFP4 experts.  `per_channel`: one decay per key channel (the KDA variant of the GLM Flash line) instead of one per head."""
    return ModelSpec(
        name="hybrid-kda-shape" if per_channel else "hybrid-gdn-shape", family="hybrid_linear", vocab=151936, hidden=2048, n_layers=n_layers, rms_eps=1e-6,
        attn=AttentionSpec(kind="gqa", n_heads=16, n_kv_heads=2, head_dim=128, rope_theta=1e6, rope_interleaved=False, qk_norm=True,
                           linear_every=4, linear_k_heads=16, linear_v_heads=32, linear_per_channel=per_channel),
        moe=MoESpec(n_experts=128, top_k=8, intermediate=768, n_shared=1, scoring="softmax", normalize=True),
        quant=QuantSpec(experts="nvfp4", dense="bf16", kv="bf16"))


def bedovik_spec(n_layers: int = 8, heads: int = 32, hidden: int = 4096, rank: int = 512, experts: int = 64, ff: int = 1536, loop_times: int = 2) -> ModelSpec:
    """Bedovik at the size of a real model's layers (synthetic weights): parallel latent-attention layers, gated and plain ones in turn,
    squared-ReLU experts behind group-limited softmax routing, the middle half of the stack looped."""
    moe = MoESpec(n_experts=experts, top_k=8, intermediate=ff, n_shared=0, scoring="softmax", normalize=True, route_scale=2.5, n_group=8, topk_group=4,
                  activation="relu2", group_score="max")
    attn = AttentionSpec(kind="latent", n_heads=heads, n_kv_heads=heads, head_dim=128, v_head_dim=128, kv_lora_rank=rank, scale=128 ** -0.5)
    blocks = tuple(BlockSpec(dataclasses.replace(attn, out_gate=i % 2 == 0), moe) for i in range(n_layers))
    lo, hi = n_layers // 4, n_layers - n_layers // 4
    return ModelSpec(name="bedovik-shape", family="bedovik", vocab=65536, hidden=hidden, n_layers=n_layers, rms_eps=1e-6, attn=blocks[0].attn, moe=moe,
                     quant=QuantSpec(experts="bf16", dense="bf16", kv="bf16"), blocks=blocks,
                     loop=LoopSpec(lo, hi, loop_times) if loop_times > 1 and hi > lo else None, learned_positions=65536, max_context=65536)


def tudilix_spec(n_layers: int = 12, hidden: int = 4096, heads: int = 32, kv_heads: int = 4, ff: int = 12288, window: int = 2048, blocks: int = 16,
                 ffn_everywhere: bool = False) -> ModelSpec:
    """Tudilix at the size of a real model's layers (synthetic weights): two recurrent layers, then one windowed-attention layer, every second
    attention layer on the keys and values of the one before it; dense feed-forwards behind the attention layers, or behind every layer."""
    rec = BlockSpec(None, rec=RecurrentSpec(width=hidden, blocks=blocks, conv_taps=4), ffn=DenseFfnSpec(ff, 7.0) if ffn_everywhere else None)
    attn = AttentionSpec(kind="conv_gqa", n_heads=heads, n_kv_heads=kv_heads, head_dim=128, v_head_dim=128, scale=128 ** -0.5, window=window, qk_norm=True, conv_taps=4,
                         rope_dims=64, rope_scaling=RopeScaling(4.0, 16384, 24.0, 1.0))
    layers, last = [], -1
    for i in range(n_layers):
        if i % 3 != 2:
            layers.append(rec)
            continue
        layers.append(BlockSpec(dataclasses.replace(attn, kv_from=last), ffn=DenseFfnSpec(ff, 7.0)))
        last = i if last < 0 else -1
    return ModelSpec(name="tudilix-shape", family="tudilix", vocab=65536, hidden=hidden, n_layers=n_layers, rms_eps=1e-6, attn=attn, moe=MoESpec(n_experts=0, n_shared=0),
                     quant=QuantSpec(experts="bf16", dense="bf16", kv="bf16"), blocks=tuple(layers), residual_mult=0.5, logit_softcap=40.0)


def vozetar_spec(n_layers: int = 6, hidden: int = 4096, heads: int = 32, kv_heads: int = 4, ff: int = 12288, window: int = 2048, rec_heads: int = 16, rec_dim: int = 128,
                 rec_vdim: int = 256, experts: int = 0, expert_ff: int = 1536, streams: int = 4, mixers: str = "PGA", moe_every: int = 2) -> ModelSpec:
    """Vozetar at the size of a real model's layers (synthetic weights).  `mixers` repeats over the layers: P windowed attention beside retention, G
    windowed attention (values are the keys) beside gated linear attention, A full attention.  `experts` > 0: routed experts (with a shared one)
    instead of a dense feed-forward in every `moe_every`-th layer."""
    base = AttentionSpec(kind="conv_gqa", n_heads=heads, n_kv_heads=kv_heads, head_dim=128, v_head_dim=128, scale=128 ** -0.5, rope_dims=128, conv_taps=0)
    windowed = dataclasses.replace(base, window=window, keep_first=4, rope_dims=64, rope_theta=1e6)
    rec = RecurrentSpec(kind="retention", heads=rec_heads, dim=rec_dim, vdim=rec_vdim, decay=tuple(1.0 - 2.0 ** (-5 - 7.0 * i / rec_heads) for i in range(rec_heads)), rope_dims=rec_dim)
    kinds = {"P": (dataclasses.replace(windowed, qkv_bias=True, sink=True), rec, (1.0, 0.8), False),
             "G": (dataclasses.replace(windowed, values_are_keys=True, conv_taps=3, qk_norm_whole=True, out_gate=True), dataclasses.replace(rec, kind="gla", decay=(), rope_dims=0, tau=16.0, rank=16),
                   (0.5, 0.5), True),
             "A": (dataclasses.replace(base, rope_interleaved=False, conv_taps=4, qkv_bias=True, out_bias=True, sink=True, out_gate=True, gate_values=True), None, (1.0, 1.0), False)}
    moe = MoESpec(n_experts=experts, top_k=8, intermediate=expert_ff, n_shared=1, shared_intermediate=expert_ff, scoring="sigmoid", normalize=False, n_group=8, topk_group=4) if experts else None
    blocks = []
    for i in range(n_layers):
        attn, r, scales, norm = kinds[mixers[i % len(mixers)]]
        routed = moe is not None and i % moe_every == moe_every - 1
        blocks.append(BlockSpec(attn, moe if routed else None, r, None if routed else DenseFfnSpec(ff, activation="silu_glu"), scales, norm))
    return ModelSpec(name="vozetar-shape", family="vozetar", vocab=65536, hidden=hidden, n_layers=n_layers, rms_eps=1e-5, attn=blocks[0].attn, moe=moe or MoESpec(n_experts=0, n_shared=0),
                     quant=QuantSpec(experts="bf16", dense="bf16", kv="bf16"), blocks=tuple(blocks), streams=streams, pair_table=PairTableSpec(65521, 40503, 9973))


def sikazen_spec(n_layers: int = 6, hidden: int = 4096, heads: int = 32, kv_heads: int = 4, ff: int = 12288, window: int = 2048, pool: int = 16, rank: int = 512, q_rank: int = 1536,
                 rec_heads: int = 16, rec_dim: int = 128, rec_vdim: int = 256, side: int = 256, mixers: str = "LHA", loop: tuple | None = None) -> ModelSpec:
    """Sikazen at the size of a real model's layers (synthetic weights).  `mixers` repeats over the layers: L rotated latent attention with sinks, H HGRN2,
    A windowed attention with pooled blocks.  `loop`: (start, stop, times)."""
    kinds = {"L": (AttentionSpec(kind="latent", n_heads=heads, n_kv_heads=heads, head_dim=128, v_head_dim=128, kv_lora_rank=rank, q_lora_rank=q_rank, rope_dims=64, rope_theta=1e6,
                                 scale=192 ** -0.5, sink=True), None),
             "H": (None, RecurrentSpec(kind="hgrn2", heads=rec_heads, dim=rec_dim, vdim=rec_vdim)),
             "A": (AttentionSpec(kind="conv_gqa", n_heads=heads, n_kv_heads=kv_heads, head_dim=128, v_head_dim=128, scale=128 ** -0.5, window=window, pool=pool, conv_taps=0, rope_dims=128,
                                 rope_interleaved=False, rope_divisor=4.0, qk_norm_unit=True, qkv_bias=True), None)}
    blocks = tuple(BlockSpec(a, rec=r, ffn=DenseFfnSpec(ff, activation="silu_glu")) for a, r in (kinds[mixers[i % len(mixers)]] for i in range(n_layers)))
    return ModelSpec(name="sikazen-shape", family="sikazen", vocab=65536, hidden=hidden, n_layers=n_layers, rms_eps=1e-5,
                     attn=next((b.attn for b in blocks if b.attn is not None), AttentionSpec(kind="conv_gqa", n_heads=1, n_kv_heads=1)), moe=MoESpec(n_experts=0, n_shared=0),
                     quant=QuantSpec(experts="bf16", dense="bf16", kv="bf16"), blocks=blocks, mixed=True, embed_scale=hidden ** 0.5, side_dim=side,
                     loop=LoopSpec(*loop, entry="add") if loop else None)


NAMED_SPECS = {
    "tiny": tiny_spec,
    "hybrid-gdn": hybrid_gdn_spec,
    "hybrid-kda": lambda **kw: hybrid_gdn_spec(per_channel=True, **kw),
    "deepseek-v3": deepseek_v3_spec,
    "deepseek-v32": deepseek_v32_spec,
    "qwen3-235b": qwen3_235b_spec,
    "bedovik": bedovik_spec,
    "tudilix": tudilix_spec,
    "vozetar": vozetar_spec,
    "sikazen": sikazen_spec,
    "ep-microbench": ep_microbench_spec,
}


def spec_by_name(name: str, **kw) -> ModelSpec:
    if name not in NAMED_SPECS:
        raise KeyError(f"unknown model spec {name!r}; known: {sorted(NAMED_SPECS)}")
    return NAMED_SPECS[name](**kw)


# ---------------------------------------------------------------------------
# HF config.json -> ModelSpec (family detection, reference: commands/family.rs)
# ---------------------------------------------------------------------------

FAMILY_BY_ARCH = {
    "DeepseekV3ForCausalLM": "deepseek_v3",
    "DeepseekV32ForCausalLM": "deepseek_v3",
    "DeepseekV4ForCausalLM": "deepseek_v4",
    "Qwen3MoeForCausalLM": "qwen3_moe",
    "Qwen3ForCausalLM": "qwen3_dense",
    "Glm4MoeForCausalLM": "glm_moe",
    "GlmMoeDsaForCausalLM": "glm_moe",
    "MiMoV2FlashForCausalLM": "mimo_v2",
    "MixtralForCausalLM": "mixtral",
    "Qwen3NextForCausalLM": "hybrid_linear",
    "Bedovik": "bedovik",
    "Tudilix": "tudilix",
    "Vozetar": "vozetar",
    "Sikazen": "sikazen",
}


def detect_quant(cfg: dict) -> QuantSpec:
    q = cfg.get("quantization_config") or {}
    method = (q.get("quant_method") or q.get("quant_algo") or "").lower()
    fmt = (q.get("fmt") or q.get("format") or "").lower()
    if method == "fp8":
        blk = q.get("weight_block_size") or [128, 128]
        dense = "fp8_block32" if list(blk) == [32, 32] else "fp8_block128"
        experts = "mxfp4" if "mxfp4" in json.dumps(q).lower() else dense
        return QuantSpec(experts=experts, dense=dense)
    if method in ("mxfp4",):
        return QuantSpec(experts="mxfp4", dense="bf16")
    if method in ("modelopt", "nvfp4") or "nvfp4" in fmt or q.get("quant_algo", "").upper() == "NVFP4":
        return QuantSpec(experts="nvfp4", dense="nvfp4")
    if method in ("exl3",) or "exl3" in fmt:
        return QuantSpec(experts="exl3", dense="bf16", exl3_bits=int(round(float(q.get("bits", 4)))))
    return QuantSpec()


def _bedovik_config(cfg: dict) -> ModelSpec:
    """`config.json` of the Bedovik design: every layer names its mixer and its feed-forward with their sizes."""
    blocks = []
    for i, layer in enumerate(cfg["layers"]):
        if layer["type"] not in ("latent_attention", "latent_attention_2"):
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        m = layer["mixer"]
        attn = AttentionSpec(kind="latent", n_heads=int(m["heads"]), n_kv_heads=int(m["heads"]), head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]),
                             kv_lora_rank=int(m["kv_rank"]), scale=float(m["scale"]), out_gate=layer["type"] == "latent_attention")
        mlp, moe = layer.get("mlp"), None
        if mlp is not None:
            if mlp.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            r = mlp["router"]
            groups = r.get("groups") or {"count": 1, "keep": 1}
            moe = MoESpec(n_experts=int(r["experts"]), top_k=int(r["top"]), intermediate=int(mlp["expert"]["ff"]), n_shared=0, scoring="softmax",
                          normalize=True, route_scale=float(r.get("scale", 1.0)), n_group=int(groups["count"]), topk_group=int(groups["keep"]),
                          activation="relu2", group_score="max")
            if moe.n_experts % moe.n_group or not 1 <= moe.topk_group <= moe.n_group or moe.top_k > moe.n_experts // moe.n_group * moe.topk_group:
                raise ValueError(f"layer {i}: {moe.n_experts} experts in {moe.n_group} groups, {moe.topk_group} kept, top {moe.top_k}: not a routing")
        blocks.append(BlockSpec(attn, moe))
    loop = None
    if cfg.get("loop"):
        loop = LoopSpec(int(cfg["loop"]["start"]), int(cfg["loop"]["stop"]), int(cfg["loop"]["times"]))
        if not (0 <= loop.start < loop.stop <= len(blocks) and loop.times >= 1):
            raise ValueError(f"loop {cfg['loop']} does not fit {len(blocks)} layers")
    n_pos = int(cfg["max_positions"])
    return ModelSpec(name="bedovik", family="bedovik", vocab=int(cfg["vocab"]), hidden=int(cfg["width"]), n_layers=len(blocks),
                     rms_eps=float(cfg["norm"]["eps"]), attn=blocks[0].attn, moe=next((b.moe for b in blocks if b.moe is not None), MoESpec(n_experts=0, n_shared=0)),
                     quant=QuantSpec(), blocks=tuple(blocks), loop=loop, learned_positions=n_pos, max_context=n_pos)


def _tudilix_config(cfg: dict) -> ModelSpec:
    """`config.json` of the Tudilix design: every layer names its mixer (windowed attention or a gated linear recurrence) and its
    feed-forward with their sizes."""
    blocks = []
    for i, layer in enumerate(cfg["layers"]):
        m, mlp = layer["mixer"], layer.get("mlp")
        attn = rec = ffn = None
        if layer["type"] == "rglru":
            rec = RecurrentSpec(width=int(m["width"]), blocks=int(m["blocks"]), conv_taps=int(m["conv"]))
            if rec.width % rec.blocks:
                raise ValueError(f"layer {i}: {rec.width} channels in {rec.blocks} blocks")
        elif layer["type"] == "attention":
            rot = m.get("rot") or {"dims": 0, "base": 1e4}
            sc = rot.get("scaling")
            attn = AttentionSpec(kind="conv_gqa", n_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]),
                                 scale=float(m["scale"]), window=int((m.get("mask") or {}).get("size") or 0), qk_norm=True, conv_taps=int(m["conv"]),
                                 rope_dims=int(rot["dims"]), rope_theta=float(rot["base"]),
                                 rope_scaling=RopeScaling(*(float(sc[k]) for k in ("factor", "original", "fast", "slow"))) if sc else None,
                                 kv_from=int(m["kv_from"]) if m.get("kv_from") is not None else -1)
            if attn.n_heads % attn.n_kv_heads:
                raise ValueError(f"layer {i}: {attn.n_heads} query heads over {attn.n_kv_heads} key heads")
            if attn.rope_dims % 2 or attn.rope_dims > attn.head_dim:
                raise ValueError(f"layer {i}: {attn.rope_dims} rotated dimensions of {attn.head_dim}")
            if attn.kv_from >= 0:
                src = blocks[attn.kv_from].attn if attn.kv_from < i else None
                if src is None or src.kv_from >= 0 or (src.n_kv_heads, src.head_dim, src.v_head_dim) != (attn.n_kv_heads, attn.head_dim, attn.v_head_dim):
                    raise ValueError(f"layer {i}: layer {attn.kv_from} has no keys and values of its shape")
        else:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            ffn = DenseFfnSpec(int(mlp["ff"]), float(mlp["limit"]))
        blocks.append(BlockSpec(attn, rec=rec, ffn=ffn))
    first = next((b.attn for b in blocks if b.attn is not None), AttentionSpec(kind="conv_gqa", n_heads=1, n_kv_heads=1))
    return ModelSpec(name="tudilix", family="tudilix", vocab=int(cfg["vocab"]), hidden=int(cfg["width"]), n_layers=len(blocks), rms_eps=float(cfg["norm"]["eps"]),
                     attn=first, moe=MoESpec(n_experts=0, n_shared=0), quant=QuantSpec(), blocks=tuple(blocks), residual_mult=float(cfg["residual_mult"]),
                     logit_softcap=float(cfg.get("logit_softcap") or 0.0))


def _vozetar_attention(i: int, m: dict, **kw) -> AttentionSpec:
    rot, mask = m.get("rot") or {"dims": 0, "base": 1e4}, m.get("mask") or {}
    a = AttentionSpec(kind="conv_gqa", n_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]), scale=float(m["scale"]),
                      window=int(mask.get("size") or 0), keep_first=int(mask.get("keep_first") or 0), conv_taps=int(m.get("conv") or 0), rope_dims=int(rot["dims"]),
                      rope_theta=float(rot["base"]), **kw)
    if a.n_heads % a.n_kv_heads:
        raise ValueError(f"layer {i}: {a.n_heads} query heads over {a.n_kv_heads} key heads")
    if a.rope_dims % 2 or a.rope_dims > a.head_dim:
        raise ValueError(f"layer {i}: {a.rope_dims} rotated dimensions of {a.head_dim}")
    if a.values_are_keys and a.v_head_dim != a.head_dim:
        raise ValueError(f"layer {i}: values are the keys, but {a.v_head_dim} is not {a.head_dim}")
    return a


def _vozetar_config(cfg: dict) -> ModelSpec:
    """`config.json` of the Vozetar design: every layer names its mixer (attention, or attention beside a linear one) and its feed-forward with
    their sizes."""
    blocks = []
    for i, layer in enumerate(cfg["layers"]):
        m, mlp, kind = layer["mixer"], layer.get("mlp"), layer["type"]
        rec, moe, ffn, scales = None, None, None, (1.0, 1.0)
        if kind == "attention":
            attn = _vozetar_attention(i, m, rope_interleaved=False, qkv_bias=True, out_bias=True, sink=True, out_gate=True, gate_values=True)
        elif kind == "parallel":
            attn = _vozetar_attention(i, m["left"], qkv_bias=True, sink=True)
            r = m["right"]
            rot = r.get("rot") or {"dims": 0, "base": 1e4}
            rec = RecurrentSpec(kind="retention", heads=int(r["heads"]), dim=int(r["dim"]), vdim=int(r["vdim"]), decay=tuple(float(x) for x in r["decay"]), rope_dims=int(rot["dims"]),
                                rope_theta=float(rot["base"]))
            if len(rec.decay) != rec.heads or rec.rope_dims % 2 or rec.rope_dims > rec.dim:
                raise ValueError(f"layer {i}: {len(rec.decay)} decays of {rec.heads} heads, {rec.rope_dims} rotated dimensions of {rec.dim}")
            scales = (float(m["left_scale"]), float(m["right_scale"]))
        elif kind == "parallel_2":
            attn = _vozetar_attention(i, m["left"], values_are_keys=True, qk_norm_whole=True, out_gate=True)
            r = m["right"]
            rec = RecurrentSpec(kind="gla", heads=int(r["heads"]), dim=int(r["dim"]), vdim=int(r["vdim"]), tau=float(r["tau"]))
            scales = (0.5, 0.5)
        else:
            raise ValueError(f"layer {i}: unknown mixer {kind!r}")
        if mlp is not None and mlp["kind"] == "dense":
            ffn = DenseFfnSpec(int(mlp["ff"]), activation="silu_glu")
        elif mlp is not None and mlp["kind"] == "moe":
            r, shared = mlp["router"], mlp.get("shared")
            groups = r.get("groups") or {"count": 1, "keep": 1}
            moe = MoESpec(n_experts=int(r["experts"]), top_k=int(r["top"]), intermediate=int(mlp["expert"]["ff"]), n_shared=1 if shared else 0,
                          shared_intermediate=int(shared["ff"]) if shared else 0, scoring="sigmoid", normalize=False, n_group=int(groups["count"]), topk_group=int(groups["keep"]))
            if moe.n_experts % moe.n_group or not 1 <= moe.topk_group <= moe.n_group or moe.top_k > moe.n_experts // moe.n_group * moe.topk_group:
                raise ValueError(f"layer {i}: {moe.n_experts} experts in {moe.n_group} groups, {moe.topk_group} kept, top {moe.top_k}: not a routing")
        elif mlp is not None:
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        blocks.append(BlockSpec(attn, moe, rec, ffn, scales, kind == "parallel_2"))
    pairs = (cfg.get("embedding") or {}).get("bigram")
    streams = int(cfg["streams"])
    if streams < 1:
        raise ValueError(f"{streams} residual streams")
    return ModelSpec(name="vozetar", family="vozetar", vocab=int(cfg["vocab"]), hidden=int(cfg["width"]), n_layers=len(blocks), rms_eps=float(cfg["norm"]["eps"]),
                     attn=blocks[0].attn, moe=next((b.moe for b in blocks if b.moe is not None), MoESpec(n_experts=0, n_shared=0)), quant=QuantSpec(), blocks=tuple(blocks),
                     streams=streams, pair_table=PairTableSpec(int(pairs["buckets"]), int(pairs["mul_prev"]), int(pairs["mul_cur"])) if pairs else None)


def _sikazen_config(cfg: dict) -> ModelSpec:
    """`config.json` of the Sikazen design: every layer names its mixer (attention with pooled blocks, rotated latent attention, HGRN2) and its
    feed-forward with their sizes."""
    blocks = []
    for i, layer in enumerate(cfg["layers"]):
        m, mlp, kind = layer["mixer"], layer.get("mlp"), layer["type"]
        attn = rec = ffn = None
        rot = m.get("rot") or {"dims": 0, "base": 1e4}
        turn = dict(rope_theta=float(rot["base"]), rope_divisor=float((rot.get("scaling") or {}).get("factor", 1.0)))
        if kind == "attention":
            mask = m.get("mask") or {}
            attn = AttentionSpec(kind="conv_gqa", n_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]), scale=float(m["scale"]),
                                 window=int(mask.get("size") or 0), pool=int(mask.get("pool") or 0) if mask.get("size") else 0, conv_taps=0, rope_dims=int(rot["dims"]),
                                 rope_interleaved=False, qk_norm_unit=True, qkv_bias=True, **turn)
            if attn.n_heads % attn.n_kv_heads:
                raise ValueError(f"layer {i}: {attn.n_heads} query heads over {attn.n_kv_heads} key heads")
            if attn.rope_dims % 2 or attn.rope_dims > attn.head_dim:
                raise ValueError(f"layer {i}: {attn.rope_dims} rotated dimensions of {attn.head_dim}")
            if attn.window < 0 or attn.pool < 0:
                raise ValueError(f"layer {i}: window of {attn.window} tokens, blocks of {attn.pool}")
        elif kind == "latent_attention":
            attn = AttentionSpec(kind="latent", n_heads=int(m["heads"]), n_kv_heads=int(m["heads"]), head_dim=int(m["dim"]), v_head_dim=int(m["vdim"]), kv_lora_rank=int(m["kv_rank"]),
                                 q_lora_rank=int(m["q_rank"]), rope_dims=int(m["rot_dim"]), scale=float(m["scale"]), sink=True, **turn)
            if attn.rope_dims % 2 or int(rot["dims"]) != attn.rope_dims:
                raise ValueError(f"layer {i}: rotation over {rot['dims']} dimensions of a rotated part of {attn.rope_dims}")
        elif kind == "hgrn2":
            rec = RecurrentSpec(kind="hgrn2", heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
        else:
            raise ValueError(f"layer {i}: unknown mixer {kind!r}")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            ffn = DenseFfnSpec(int(mlp["ff"]), activation="silu_glu")
        blocks.append(BlockSpec(attn, rec=rec, ffn=ffn))
    loop = None
    if cfg.get("loop"):
        loop = LoopSpec(int(cfg["loop"]["start"]), int(cfg["loop"]["stop"]), int(cfg["loop"]["times"]), "add")
        if not (0 <= loop.start < loop.stop <= len(blocks) and loop.times >= 1):
            raise ValueError(f"loop {cfg['loop']} does not fit {len(blocks)} layers")
    first = next((b.attn for b in blocks if b.attn is not None), AttentionSpec(kind="conv_gqa", n_heads=1, n_kv_heads=1))
    return ModelSpec(name="sikazen", family="sikazen", vocab=int(cfg["vocab"]), hidden=int(cfg["width"]), n_layers=len(blocks), rms_eps=float(cfg["norm"]["eps"]), attn=first,
                     moe=MoESpec(n_experts=0, n_shared=0), quant=QuantSpec(), blocks=tuple(blocks), mixed=True, embed_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)),
                     side_dim=int((cfg.get("token_side") or {}).get("dim") or 0), loop=loop)


def from_hf_config(cfg: dict | str | Path) -> ModelSpec:
    """Build a ModelSpec from a Hugging Face `config.json` (dict or path)."""
    if not isinstance(cfg, dict):
        p = Path(cfg)
        p = p / "config.json" if p.is_dir() else p
        cfg = json.loads(p.read_text())
    archs = cfg.get("architectures") or [cfg.get("architecture", "?")]
    family = FAMILY_BY_ARCH.get(archs[0])
    if family is None:
        raise ValueError(f"unsupported architecture {archs[0]!r} (supported: {sorted(FAMILY_BY_ARCH)})")
    if family == "bedovik":
        return _bedovik_config(cfg)
    if family == "tudilix":
        return _tudilix_config(cfg)
    if family == "vozetar":
        return _vozetar_config(cfg)
    if family == "sikazen":
        return _sikazen_config(cfg)
    hidden = cfg["hidden_size"]
    heads = cfg["num_attention_heads"]
    if "kv_lora_rank" in cfg:
        attn = AttentionSpec(kind="mla", n_heads=heads, n_kv_heads=heads,
                             head_dim=cfg["qk_nope_head_dim"] + cfg["qk_rope_head_dim"],
                             rope_theta=cfg.get("rope_theta", 1e4),
                             q_lora_rank=cfg.get("q_lora_rank") or 0, kv_lora_rank=cfg["kv_lora_rank"],
                             qk_nope_head_dim=cfg["qk_nope_head_dim"], qk_rope_head_dim=cfg["qk_rope_head_dim"],
                             v_head_dim=cfg["v_head_dim"],
                             # sparse attention with a learned indexer (the V3.2 / GLM-5 line)
                             index_topk=cfg.get("index_topk") or 0, index_heads=cfg.get("index_n_heads") or 0,
                             index_dim=cfg.get("index_head_dim") or 0)
    else:
        attn = AttentionSpec(kind="gqa", n_heads=heads, n_kv_heads=cfg.get("num_key_value_heads", heads),
                             head_dim=cfg.get("head_dim") or hidden // heads,
                             rope_theta=cfg.get("rope_theta", 1e4), rope_interleaved=False,
                             qk_norm=family in ("qwen3_moe", "qwen3_dense"),
                             window=cfg.get("sliding_window_size") or cfg.get("sliding_window") or 0)
        if cfg.get("full_attention_interval") and cfg.get("linear_num_value_heads"):
            # hybrid linear-attention stack (the Qwen-Next line): gated delta-rule layers, every n-th layer full attention
            if cfg.get("linear_key_head_dim", 128) != 128 or cfg.get("linear_value_head_dim", 128) != 128 or cfg.get("linear_conv_kernel_dim", 4) != 4:
                raise ValueError("linear-attention layers: 128-wide key / value heads and a width-4 convolution are supported")
            attn = dataclasses.replace(attn, linear_every=int(cfg["full_attention_interval"]), linear_k_heads=int(cfg["linear_num_key_heads"]),
                                       linear_v_heads=int(cfg["linear_num_value_heads"]), qk_norm=True)
        pattern = cfg.get("hybrid_layer_pattern")            # MiMo-V2: 0 = full attention, 1 = sliding window (+ sinks)
        if attn.linear_every:
            pattern = None                                    # `layer_types` then names the linear layers, not sliding windows
        if pattern is None and cfg.get("layer_types") and not attn.linear_every:
            pattern = [0 if t == "full_attention" else 1 for t in cfg["layer_types"]]
        if pattern and any(pattern):
            full = [i for i, p in enumerate(pattern) if not p]
            period = (full[1] - full[0]) if len(full) > 1 else len(pattern)
            if not full or full[0] != 0 or any(bool(p) == (i % period == 0) for i, p in enumerate(pattern)):
                raise ValueError("unsupported layer pattern: full-attention layers must sit at layer 0 and every n-th layer after it")
            attn = dataclasses.replace(attn, full_every=period, swa_rope_theta=float(cfg.get("swa_rope_theta") or 0.0),
                                       sink=bool(cfg.get("add_swa_attention_sink_bias", True)))
    n_exp = cfg.get("n_routed_experts") or cfg.get("num_experts") or cfg.get("num_local_experts") or 0
    moe = MoESpec(
        n_experts=n_exp, top_k=cfg.get("num_experts_per_tok", 1),
        intermediate=cfg.get("moe_intermediate_size") or cfg.get("intermediate_size", 0),
        n_shared=cfg.get("n_shared_experts") or 0,
        scoring=cfg.get("scoring_func", "softmax"), normalize=cfg.get("norm_topk_prob", True),
        route_scale=cfg.get("routed_scaling_factor", 1.0),
        use_bias=cfg.get("topk_method") == "noaux_tc", n_group=cfg.get("n_group") or 1,
        topk_group=cfg.get("topk_group") or 1, first_dense=cfg.get("first_k_dense_replace", 0),
        dense_intermediate=cfg.get("intermediate_size", 0))
    return ModelSpec(name=cfg.get("_name_or_path") or family, family=family, vocab=cfg["vocab_size"],
                     hidden=hidden, n_layers=cfg["num_hidden_layers"], rms_eps=cfg.get("rms_norm_eps", 1e-6),
                     attn=attn, moe=moe, quant=detect_quant(cfg),
                     mtp_layers=cfg.get("num_nextn_predict_layers", 0),
                     tie_embeddings=cfg.get("tie_word_embeddings", False),
                     max_context=cfg.get("max_position_embeddings", 1 << 20))


SPEC_FILE = "cuteafd_spec.json"


def spec_to_json(spec: ModelSpec) -> dict:
    """Lossless dump of a model spec (written next to synthetic snapshots, whose shapes have no Hugging Face architecture)."""
    return dataclasses.asdict(spec)


def spec_from_json(d: dict) -> ModelSpec:
    d = dict(d)
    if "engram_layers" in d:
        d["engram_layers"] = tuple(d["engram_layers"])
    def attn(a: dict) -> AttentionSpec:
        return AttentionSpec(**dict(a, rope_scaling=RopeScaling(**a["rope_scaling"]) if a.get("rope_scaling") else None))

    def block(b: dict) -> BlockSpec:
        part = lambda key, make: make(b[key]) if b.get(key) else None
        return BlockSpec(part("attn", attn), part("moe", lambda m: MoESpec(**m)), part("rec", lambda r: RecurrentSpec(**dict(r, decay=tuple(r.get("decay") or ())))),
                         part("ffn", lambda f: DenseFfnSpec(**f)), tuple(b.get("merge_scales") or (1.0, 1.0)), bool(b.get("merge_norm")))

    if d.get("blocks"):
        d["blocks"] = tuple(block(b) for b in d["blocks"])
    d["blocks"] = tuple(d.get("blocks") or ())
    if d.get("loop"):
        d["loop"] = LoopSpec(**d["loop"])
    if d.get("pair_table"):
        d["pair_table"] = PairTableSpec(**d["pair_table"])
    return ModelSpec(attn=attn(d.pop("attn")), moe=MoESpec(**d.pop("moe")), quant=QuantSpec(**d.pop("quant")), **d)


def spec_from_snapshot(path: str | Path) -> ModelSpec:
    """Model spec of a snapshot directory: the native spec file when the snapshot has one, else its `config.json`."""
    p = Path(path)
    if (p / SPEC_FILE).exists():
        return spec_from_json(json.loads((p / SPEC_FILE).read_text()))
    return from_hf_config(p)


@dataclass(frozen=True)
class Deployment:
    """How ranks of one node are used (reference: SparkWorld / placement decisions).

    attention ranks run attention + dense backbone + router + shared expert (+ head);
    expert ranks hold routed experts, expert-parallel.  With `colocated=True` every rank does both."""
    world: int = 1
    attn_ranks: tuple = (0,)
    expert_ranks: tuple = (0,)
    colocated: bool = True
    attn_groups: int = 1        # data-parallel attention groups; each group is `tp` consecutive entries of attn_ranks

    @property
    def tp(self) -> int:
        return len(self.attn_ranks) // max(1, self.attn_groups)

    @property
    def ep(self) -> int:
        return len(self.expert_ranks)

    def group_of(self, rank: int) -> int:
        return self.attn_ranks.index(rank) // self.tp

    def group_ranks(self, g: int) -> tuple:
        return tuple(self.attn_ranks[g * self.tp:(g + 1) * self.tp])

    def describe(self) -> str:
        if self.world == 1:
            return "single"
        dp = f"dp{self.attn_groups}x" if self.attn_groups > 1 else ""
        return f"attn-{dp}tp{self.tp}+ep{self.ep}" if not self.colocated else f"colocated attn-{dp}tp{self.tp} + ep{self.ep} on the same GPUs"


def default_deployment(world: int, attn_groups: int = 1) -> Deployment:
    """North-star split: attention TP2 on ranks 0-1, experts EP on the rest (8 GPUs -> TP2 + EP6).  With
    `attn_groups` > 1 the attention side is that many data-parallel groups (each serving its own sequences, all
    sending to the same expert ranks, which work on one group's tokens while the other groups run attention):
    4 GPUs -> 2 x TP1 + EP2, 8 GPUs -> 2 x TP2 + EP4."""
    if world == 1:
        return Deployment()
    if world == 2:
        return Deployment(world=2, attn_ranks=(0,), expert_ranks=(1,), colocated=False)
    if attn_groups <= 1:
        return Deployment(world=world, attn_ranks=(0, 1), expert_ranks=tuple(range(2, world)), colocated=False)
    n_attn = max(attn_groups, (world // 2 // attn_groups) * attn_groups)
    if n_attn >= world:
        raise ValueError(f"{attn_groups} attention groups leave no expert rank in a world of {world}")
    return Deployment(world=world, attn_ranks=tuple(range(n_attn)), expert_ranks=tuple(range(n_attn, world)), colocated=False,
                      attn_groups=attn_groups)


def colocated_deployment(world: int) -> Deployment:
    """Every GPU is an attention rank for its own sequences (data-parallel attention, TP1) AND an expert rank for its share
    of the routed experts (reference counterpart: routed layers resident on the coordinator GPUs, `--rtx-expert-layers`,
    shared/experts/local.rs; on NVSwitch every GPU can afford both roles)."""
    if world == 1:
        return Deployment()
    ranks = tuple(range(world))
    return Deployment(world=world, attn_ranks=ranks, expert_ranks=ranks, colocated=True, attn_groups=world)


def deployment_by_name(layout: str, world: int, attn_groups: int = 1) -> Deployment:
    """`split` = disjoint attention / expert ranks (`default_deployment`), `colocated` = both roles on every GPU."""
    if layout == "colocated":
        return colocated_deployment(world)
    if layout == "split":
        return default_deployment(world, attn_groups)
    raise ValueError(f"unknown layout {layout!r} (split | colocated)")

"""Engine of latent-attention layer stacks (the Bedovik design): unequal parallel layers over an fp32 residual, a looped layer range,
latent attention without positions, squared-ReLU experts.

Runs the generic engine's steps (packed inputs, paged cache, CUDA graphs per shape, head and token selection) with its own layer program:

  token + position rows -> x (fp32)
  per layer run   [at the start of a pass: x = W_in [x; x0], x += step vector]
                  h = tanh(alpha x) w + b                              written by whichever kernel produced x
                  h -> queries | latent | gates | router logits        one product, fp32 output
                  latent_prepare                                       cache row, head-major queries, gates, logits
                  decode: q W_uk -> absorbed attention over the latent pages -> W_uv (token-major) -> W_o
                  prefill chunks: context rows -> keys / values (one product) -> per-head attention -> W_o
                  routing + packing -> gather -> W_up (squared ReLU in the epilogue) -> W_down
                  x += ls1 * mixer + ls2 * experts, next h or next [x; x0]     one launch
  rows that need logits -> final norm -> head

The cache holds one latent row per token and layer RUN (a looped layer keeps one per pass), all runs in one store of a common row width, so
page bookkeeping, prefix sharing and the host tier treat it like any other paged cache.  With fp32 weights (`QuantSpec.dense = "f32"`) the
same program runs entirely in fp32: fp32 products, the ordinary-core attention kernel, an fp32 cache.
"""
from __future__ import annotations

import torch

from .. import ops
from ..models.latent_stack import StackLayer, StackWeights, up
from ..ops import ActBuffer, KIND_BF16, native
from ..ops.native import call, ptr, stream
from .engine import PAGE, StepShape
from .mla import MlaEngine
from .stack import StackBase, StackLane


class LatentLane(StackLane):
    def __init__(self, eng: "LatentStackEngine", cap: int):
        super().__init__(eng, cap)
        self.cat = self.cat_act = None
        if eng.spec.loop is not None:
            self.cat, self.cat_act = self._operand(cap, 2 * eng.Wp)

    def mixer(self, a, n_in: int) -> dict:
        """Buffers of one mixer geometry (head-major buffers are [heads, cap, .]: head h of row t is row h * cap + t)."""
        H, dp, rp, cap = a.n_heads, up(a.head_dim, 64), up(a.kv_lora_rank, 64), self.cap

        def make():
            q, q_act = self._operand(H * cap, dp)
            o, o_act = self._operand(cap, up(H * a.v_head_dim, 8))
            return {"proj": torch.zeros(cap, up(n_in, 8), dtype=torch.float32, device=self.dev), "q": q, "q_act": q_act, "o": o, "o_act": o_act,
                    "gate": torch.zeros(cap, H, dtype=torch.float32, device=self.dev),
                    "tiles": torch.zeros(H * -(-cap // self.tn), 4, dtype=torch.int32, device=self.dev),
                    "n_tiles": torch.zeros(1, dtype=torch.int32, device=self.dev), "max_tiles": H * -(-cap // self.tn)}
        return self.get(("mix", H, a.head_dim, a.v_head_dim, rp, n_in), make)


class LatentAttention:
    """Attention over paged latent rows, for engines on `StackBase`: absorbed over the rows themselves (decoding, short runs, fp32), or - long runs -
    per head over keys and values that the context's rows are expanded to.  Optional: a rotated part behind the latent (`AttentionSpec.rope_dims`;
    queries' parts in b["qr"]), sinks, output gates.  `b`: the lane's buffers (`q` head-major unrotated queries, `o` attended rows, `tiles`)."""
    _ctx_plan = MlaEngine._ctx_plan
    PREFILL_MAX_BYTES = MlaEngine.PREFILL_MAX_BYTES

    @property
    def latent_prefill_min_q(self) -> int:
        """Query rows of a sequence from which the context is expanded (0: never)."""
        return MlaEngine.PREFILL_MIN_Q

    def _latent_fill(self, a, n_seq: int, max_q_len: int) -> int:
        """Splits of a layer's absorbed attention that fill the machine once."""
        rp, H = up(a.kv_lora_rank, 64), a.n_heads
        ctas = (1 if rp <= 256 else 2) * n_seq * -(-max_q_len // max(1, 128 // min(H, 128)))
        return max(1, self.sm_count * (2 if rp <= 128 else 1) // ctas)            # narrow latents: two CTAs per SM

    def _latent_splits(self, a, n_seq: int, max_q_len: int, max_kv: int) -> int:
        tiles, fill = max(1, -(-max_kv // PAGE)), self._latent_fill(a, n_seq, max_q_len)
        if tiles < min(32, fill):
            return 1 << (tiles.bit_length() - 1)       # short contexts: powers of two, so a growing context re-captures rarely
        return max(1, min(32, fill))

    def _latent_maps(self, planes: torch.Tensor, attns: list) -> torch.Tensor:
        """TMA descriptors of the planes [., slots, row] of layers of these kinds."""
        host = torch.zeros(len(attns), 128, dtype=torch.uint8)
        for r, a in enumerate(attns):
            call("cuteafd_tmap_encode_latent_rows", host[r].data_ptr(), planes[r].data_ptr(), planes.shape[1], a.latent_row, planes.shape[2])
        return host.to(self.device)

    def _latent_attention(self, a, lw, L, b: dict, rows: torch.Tensor, tmap, gate, sh: StepShape):
        if self._expands(a, sh):
            self._expanded(a, lw, L, b, rows, gate, sh)
        else:
            self._absorbed(a, lw, L, b, rows, tmap, gate, sh)

    def _absorbed(self, a, lw, L, b: dict, rows: torch.Tensor, tmap, gate, sh: StepShape):
        T, md, H, rp = sh.T, self.md, a.n_heads, up(a.kv_lora_rank, 64)
        lat = L.latent(H, rp)
        per = dict(tiles=b["tiles"], n_tiles=b["n_tiles"], max_tiles=H * -(-T // L.tn), status=self.status)
        ops.tc_linear(lw.w_uk_t, b["q_act"], lat["q"], rows=H * L.cap, **per)
        common = dict(T=T, ldt=L.cap, n_seq=sh.n_seq, H=H, rank_pad=rp, scale=a.softmax_scale, q_rope=b.get("qr"), sink=lw.sink, status=self.status)
        where = (md["page_table"], md["kv_len"], md["q_start"], md["q_len"], gate, lat["o"])
        if self.f32 or rp > 512 or H > 128 or a.rope_dims > 64:
            ops.latent_attention_simt(lat["q"], rows, *where, **common)
        else:
            splits = min(sh.attn_splits, self._latent_fill(a, sh.n_seq, sh.max_q_len))
            if splits > 1:
                self._scratch(splits * T * H * rp, splits * T * H * 2)
                self.launches_per_step += 1
            ops.latent_attention(lat["q"], tmap, *where, max_q_len=sh.max_q_len, n_splits=splits, part_o=self.part_o if splits > 1 else None,
                                 part_ml=self.part_ml if splits > 1 else None, **common)
        ops.tc_linear(lw.w_uv, lat["o_act"], b["o"], rows=H * L.cap, token_major=(L.cap, a.v_head_dim), **per)
        self.launches_per_step += 3

    def _expands(self, a, sh: StepShape) -> bool:
        """Chunks whose longest query run fills a 128-row tile expand the context into per-head keys and values (see `MlaEngine`)."""
        least = self.latent_prefill_min_q
        if self.f32 or not least or sh.max_q_len < least or sh.uniform or a.head_dim > 192 or a.v_head_dim > 128 or a.rope_dims > 64:
            return False
        if torch.cuda.is_current_stream_capturing():
            return False
        rows = sum(-(-n // 64) * 64 for n in self.mh["kv_len"][:sh.n_seq].tolist()) + 64
        return rows * (a.latent_row + a.n_heads * (up(a.head_dim, 64) + up(a.v_head_dim, 64))) * 2 <= self.PREFILL_MAX_BYTES

    def _pf_buffers(self, rows: int, rp: int, row: int, width: int):
        """Context rows and their expansion (zero-filled: rows no gather ever wrote are multiplied by zero probabilities)."""
        cap, lat, act = self._pf.get(("lat", rp, row), (0, None, None))
        if rows + 64 > cap:
            cap = max(1024, 1 << (rows + 64 - 1).bit_length())
            lat = torch.zeros(cap, row, dtype=torch.bfloat16, device=self.device)
            view = lat[:, :rp]
            act = ActBuffer(KIND_BF16, cap, rp, 256, view, ops.encode_tmap(view, 256))
            self._pf[("lat", rp, row)] = (cap, lat, act)
        kcap, kvb = self._pf.get(("kvb", width), (0, None))
        if kcap < cap:
            kvb = torch.zeros(cap, width, dtype=torch.bfloat16, device=self.device)
            self._pf[("kvb", width)] = (cap, kvb)
        return cap, lat, act, kvb

    def _expanded(self, a, lw, L, b: dict, rows_: torch.Tensor, gate, sh: StepShape):
        T, md, H, n_seq = sh.T, self.md, a.n_heads, sh.n_seq
        rp, dp, dvp, row = up(a.kv_lora_rank, 64), up(a.head_dim, 64), up(a.v_head_dim, 64), a.latent_row
        kv, rows = self._ctx_plan(sh)
        cap, lat, act, kvb = self._pf_buffers(rows, rp, row, H * (dp + dvp))
        st = ptr(self.status)
        call("cuteafd_latent_gather_ctx", ptr(rows_), ptr(md["page_table"]), ptr(self._pf_starts), ptr(md["kv_len"]), ptr(lat), n_seq, max(kv),
             md["page_table"].shape[1], rows_.shape[0], cap, row, rows_.stride(0), st, stream())
        ops.tc_linear(lw.ensure_kvb(), act, kvb, rows=rows, status=self.status)
        call("cuteafd_latent_prefill_attention", ptr(b["q"]), ptr(b.get("qr")), ptr(kvb), ptr(lat), row, rp, ptr(lw.sink), cap, ptr(self._pf_starts), ptr(md["kv_len"]), ptr(md["q_start"]),
             ptr(md["q_len"]), ptr(gate), ptr(b["o"]), T, L.cap, n_seq, sh.max_q_len, H, dp, dvp, a.v_head_dim, b["o"].stride(0), a.softmax_scale, st, stream())
        self.launches_per_step += 3


class LatentStackEngine(LatentAttention, StackBase, MlaEngine):
    LANE = LatentLane

    @property
    def latent_prefill_min_q(self) -> int:
        return self.PREFILL_MIN_Q

    def __init__(self, weights: StackWeights, **kw):
        spec = weights.spec
        if spec.stack != "latent":
            raise ValueError("LatentStackEngine runs latent-attention stacks described by ModelSpec.blocks")
        self.runs = spec.layer_runs()
        for i, b in enumerate(spec.blocks):
            if b.attn.kv_lora_rank > 1024:
                raise ValueError(f"layer {i}: latents of up to 1024 values (got {b.attn.kv_lora_rank})")
            if b.moe is not None and (b.moe.n_experts > 512 or b.moe.top_k > 16 or b.moe.n_group > 32):
                raise ValueError(f"layer {i}: at most 512 experts, 16 per token, 32 groups")
        super().__init__(weights, **kw)

    # ------------------------------------------------------------------ cache
    def _alloc_attention_state(self):
        spec, n = self.spec, self.n_pages * PAGE
        self.row = max(up(b.attn.kv_lora_rank, 64) for b in spec.blocks)
        # [layer runs, slots, row]: zero-filled, so a latent's pad and slots nobody wrote hold finite values
        self.kv = torch.zeros(len(self.runs), n, self.row, dtype=torch.float32 if self.f32 else torch.bfloat16, device=self.device)
        self.kv_tmaps = None
        if not self.f32:
            self.kv_tmaps = self._latent_maps(self.kv, [spec.blocks[li].attn for li, _ in self.runs])
        self._pf: dict = {}

    def set_inputs(self, tokens, positions, *args, **kw):
        n = self.spec.learned_positions
        if n and len(positions) and max(positions) >= n:
            raise ValueError(f"position {max(positions)} is beyond this model's {n} learned positions")
        return super().set_inputs(tokens, positions, *args, **kw)

    def attn_splits_for(self, n_seq: int, max_q_len: int, max_kv: int) -> int:
        if self.f32 or max_q_len > 16:
            return 1
        return max(self._latent_splits(b.attn, n_seq, max_q_len, max_kv) for b in self.spec.blocks)

    # ------------------------------------------------------------------ layer program
    def _emit(self, r: int, L: LatentLane):
        """What the producer of the residual rows in front of layer run `r` leaves for it."""
        if r >= len(self.runs):
            return None
        li, opens = self.runs[r]
        return ops.emit_arg(cat=L.cat) if opens is not None else ops.emit_arg(norm=self.weights.layer(li).norm, xn=L.xn)

    def _forward_single(self, sh: StepShape) -> LatentLane:
        w, T, md = self.weights, sh.T, self.md
        L = self.lane(T)
        self.launches_per_step = 0
        if sh.n_logits > L.logits.shape[0]:
            L.ensure_logits(sh.n_logits)
        none = native.EmitArg()
        ops.stack_embed(md["tokens"], md["positions"], w.embed, w.pos, L.x, L.cat[:, self.Wp:] if L.cat is not None else None, self._emit(0, L) or none, T,
                        f32=self.f32, status=self.status)
        for r, (li, opens) in enumerate(self.runs):
            lw = w.layer(li)
            if opens is not None:
                self._dense(w.loop_in, L.cat_act, L.x, T)
                ops.stack_stream(L.x, ops.emit_arg(norm=lw.norm, xn=L.xn), T, f32=self.f32, vec=w.loop_step[opens])
                self.launches_per_step += 1
            self._block(r, li, lw, L, sh)
            if self.tap is not None:
                self.tap.append(L.x[:T, :self.spec.hidden].clone())
        self.launches_per_step += 1
        if sh.n_logits:
            ops.stack_stream(L.x, ops.emit_arg(norm=(w.final_norm, w.final_b, w.final_alpha), xn=L.xln), sh.n_logits, f32=self.f32, src_rows=md["logit_rows"])
            ops.tc_linear(w.lm_head, L.head_operand(sh.n_logits), L.logits, rows=sh.n_logits, status=self.status)
            ops.argmax_rows(L.logits, L.next_tok, rows=sh.n_logits, status=L.tok_status)
            self.launches_per_step += 3
        return L

    def _block(self, r: int, li: int, lw: StackLayer, L: LatentLane, sh: StepShape):
        """One parallel layer: mixer and experts read the same rows L.xn; the combine adds both to the residual and prepares run r + 1."""
        b, T = self.spec.blocks[li], sh.T
        e = L.experts(b.moe) if b.moe is not None else None
        self._mixer(r, b.attn, lw, L, sh, e)
        if e is not None:
            self._experts(b.moe, lw, L, e, T)
        ops.stack_combine(L.x, L.mix, lw.ls1, e["y"] if e else None, e["slot"] if e else None, e["wts"] if e else None, lw.ls2, self._emit(r + 1, L), T,
                          b.moe.top_k if e else 0)
        self.launches_per_step += 1

    def _mixer(self, r: int, a, lw: StackLayer, L: LatentLane, sh: StepShape, e: dict | None):
        T, md, H, rp, st = sh.T, self.md, a.n_heads, up(a.kv_lora_rank, 64), self.status
        b = L.mixer(a, lw.w_in.N)
        self._dense(lw.w_in, L.xn_act, b["proj"], T)
        gate = b["gate"] if a.out_gate else None
        ops.latent_prepare(b["proj"], lw.kv_norm, md["slot_map"], b["q"], self.kv[r], gate, e["logits"] if e else None, b["tiles"], b["n_tiles"],
                           T=T, ldt=L.cap, H=H, d=a.head_dim, r=a.kv_lora_rank, rp=rp, E=e["logits"].shape[1] if e else 0, tn=L.tn, eps=self.spec.rms_eps,
                           status=st)
        self.launches_per_step += 1
        self._latent_attention(a, lw, L, b, self.kv[r], self.kv_tmaps[r] if self.kv_tmaps is not None else None, gate, sh)
        self._dense(lw.wo, b["o_act"], L.mix, T)

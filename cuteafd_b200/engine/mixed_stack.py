"""Engine of mixed stacks (the Sikazen design): parallel layers over an fp32 residual whose mixer is attention with pooled blocks, rotated latent
attention or HGRN2; a looped layer range; a second token table behind every layer.

Runs the generic engine's steps (packed inputs, paged cache, state slots, CUDA graphs per shape, head and token selection) with its own layer
program; every arrow between two products is one launch:

  scale * token row -> x (fp32), h = x / rms(x)
  attention      h -> queries | keys | values (times the layer's number)                                             one product
                 conv_qkv: bias, rotation, unit norms -> query rows, paged cache rows, completed blocks
                 (prompts: pool_kv, the blocks that long runs complete)
                 paged attention over pooled blocks and window -> columns of the output operand
  latent         h -> queries' latent | latent, rotated key part                                                     one product, fp32 output
                 latent_down: norms, rotation -> operand of W_uq, paged cache rows;  W_uq;  latent_split: rotation, head-major queries
                 decoding: q W_uk -> absorbed attention over the latent pages -> W_uv -> columns of the output operand
                 prompts: context rows -> keys / values (one product) -> per-head attention
  HGRN2          h -> queries | forget gates | values                                                                one product
                 decay_scan: gates, recurrence, output norm -> columns of the output operand (prompts: four launches, in chunks)
  feed-forward   h -> SwiGLU in the product's epilogue (times the layer's other number) -> the columns behind the mixer's
  W_o            both side by side: mixer + feed-forward in one product
  x += that, x as operand -> W_gate -> gelu(.) * token's part of the table -> W_proj -> x += norm(.) (+ embedding output at a pass's start), next h
  rows that need logits: h -> head (times the last number)

Keys and values, pooled blocks and latents live in planes per layer RUN over the same pages; pooled rows stand with the pages of their tokens (see
`csrc/attn_extras.cuh`).  HGRN2 states live in the sequence's state slot, two per head and run, tagged with their positions (see
`csrc/decay_scan.cu`): a slot needs no reset, a repeated step repeats its writes, and up to `state_depth` tokens can be taken back by continuing
from an earlier position; blocks that tokens taken back have completed are left again before anything sees them.  With fp32 weights
(`QuantSpec.dense = "f32"`) the same program runs entirely in fp32.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config import BlockSpec
from ..models.hybrid_stack import rope_key
from ..models.latent_stack import up
from ..models.mixed_stack import MixedLayer, check_blocks, mixer_width
from .engine import PAGE, StepShape
from .hybrid_stack import HybridStackEngine
from .hyper_stack import HyperLane
from .latent_stack import LatentAttention


class MixedLane(HyperLane):
    def __init__(self, eng: "MixedStackEngine", cap: int):
        super().__init__(eng, cap)
        sd = eng.spec.side_dim
        if sd:
            self.raw, self.raw_act = self._operand(cap, eng.Wp)
            self.side_z = torch.zeros(cap, up(sd, 8), dtype=torch.float32, device=self.dev)
            self.side_g, self.side_act = self._operand(cap, up(sd, 8))

    def output(self, b: BlockSpec) -> dict:
        """The output projection's operand: the mixer's columns, then the feed-forward's."""
        K1, K2 = up(mixer_width(b), 8), up(b.ffn.intermediate, 8) if b.ffn is not None else 0

        def make():
            o, act = self._operand(self.cap, K1 + K2)
            return {"o": o[:, :K1], "h": o[:, K1:], "act": act,
                    **({"g": torch.zeros(self.cap, K2, device=self.dev), "u": torch.zeros(self.cap, K2, device=self.dev)} if self.eng.f32 and K2 else {})}
        return self.get(("out", mixer_width(b), K2), make)

    def mixer(self, b: BlockSpec, n_in: int) -> dict:
        """Buffers of one mixer geometry (head-major buffers are [heads, cap, .]: head h of row t is row h * cap + t)."""
        a, cap, dev = b.attn, self.cap, self.dev
        if a is None:
            return self.get(("hgrn2", n_in), lambda: {"proj": torch.zeros(cap, up(n_in, 8), dtype=self.dt, device=dev)})
        H, dp = a.n_heads, up(a.head_dim, 64)

        def attention():
            return {"proj": torch.zeros(cap, up(n_in, 8), dtype=self.dt, device=dev), "q": torch.zeros(cap, H * dp, dtype=self.dt, device=dev)}

        def latent():
            cq, cq_act = self._operand(cap, up(a.q_lora_rank, 8))
            q, q_act = self._operand(H * cap, dp)
            per = H * -(-cap // self.tn)
            return {"proj": torch.zeros(cap, up(n_in, 8), dtype=torch.float32, device=dev), "cq": cq, "cq_act": cq_act, "q": q, "q_act": q_act,
                    "qx": torch.zeros(cap, up(H * (a.head_dim + a.rope_dims), 8), dtype=self.dt, device=dev),
                    "qr": torch.zeros(H * cap, up(a.rope_dims, 64), dtype=self.dt, device=dev) if a.rope_dims else None,
                    "tiles": torch.zeros(per, 4, dtype=torch.int32, device=dev), "n_tiles": torch.zeros(1, dtype=torch.int32, device=dev)}
        return self.get(("mix", a.kind, H, a.head_dim, a.rope_dims, a.q_lora_rank, n_in), attention if a.kind == "conv_gqa" else latent)


class MixedStackEngine(LatentAttention, HybridStackEngine):
    LANE = MixedLane

    def _check(self, spec):
        if spec.stack != "mixed":
            raise ValueError("MixedStackEngine runs mixed stacks described by ModelSpec.blocks")
        check_blocks(spec)

    # ------------------------------------------------------------------ cache and state
    def _alloc_attention_state(self):
        from ..utils.memory_ledger import LEDGER
        spec, n, dev = self.spec, self.n_pages * PAGE, self.device
        dt = torch.float32 if self.f32 else torch.bfloat16
        self.runs = spec.layer_runs()
        attn = {r: spec.blocks[li].attn for r, (li, _) in enumerate(self.runs)}
        keyed, latent = spec.attention_runs("conv_gqa"), spec.attention_runs("latent")
        # zero-filled: pads and slots nobody wrote hold finite values
        self.kv = torch.zeros(len(keyed), n, max(64, spec.kv_row_elems()), dtype=dt, device=dev)
        self.latents = torch.zeros(len(latent), n, max(64, spec.latent_row_elems()), dtype=dt, device=dev)
        self.plane = {r: i for i, r in enumerate(keyed)} | {r: i for i, r in enumerate(latent)}
        self.pooled, self.pool_maps, self.maps = {}, {}, {}
        for r in keyed:
            a = attn[r]
            heads = (a.n_kv_heads, up(a.head_dim, 64), up(a.v_head_dim, 64))
            if a.pool:
                self.pooled[r] = torch.zeros(self.n_pages * a.pooled_page_rows, heads[0] * (heads[1] + heads[2]), dtype=dt, device=dev)
            if not self.f32:
                self.maps[self.plane[r]] = ops.encode_window_maps(self.kv[self.plane[r]], *heads)
                if a.pool:
                    self.pool_maps[r] = ops.encode_window_maps(self.pooled[r], *heads, box_rows=8)
        self.kv_tmaps = self._latent_maps(self.latents, [attn[r] for r in latent]) if latent and not self.f32 else None
        self.rings, self._pf = [None] * len(self.runs), {}
        self._alloc_states()
        with LEDGER.scope("kv"):
            LEDGER.charge(sum(t.numel() * t.element_size() for t in self.cache_buffers()[1:] + self.state_buffers()), "latents, pooled blocks, sequence state slots")

    def _alloc_states(self):
        n, D, dev = self.max_seqs, self.state_depth, self.device
        f32 = lambda *s: torch.zeros(*s, dtype=torch.float32, device=dev)
        self.states = []            # per layer run: (two states per head, their positions, inputs of the last tokens)
        for r in (self.spec.blocks[li].rec for li, _ in self.runs):
            vp = up(r.vdim, 4) if r is not None else 0
            self.states.append((f32(n, 2, r.heads, r.dim, vp), torch.zeros(n, r.heads, 2, dtype=torch.int32, device=dev), f32(n, D, r.heads, 2 * r.dim + vp))
                               if r is not None else None)

    def state_buffers(self) -> list:
        return [t for s in self.states if s is not None for t in s]

    def cache_buffers(self) -> list:
        return [self.kv, self.latents, *self.pooled.values()]

    def attn_splits_for(self, n_seq: int, max_q_len: int, max_kv: int) -> int:
        best = super().attn_splits_for(n_seq, max_q_len, max_kv)
        if self.f32 or max_q_len > 16:
            return best
        return max([best] + [self._latent_splits(b.attn, n_seq, max_q_len, max_kv) for b in self.spec.blocks if b.attn is not None and b.attn.kind == "latent"])

    # ------------------------------------------------------------------ layer program
    def _forward_single(self, sh: StepShape) -> MixedLane:
        w, spec, T, md = self.weights, self.spec, sh.T, self.md
        L = self.lane(T)
        if sh.n_logits > L.logits.shape[0]:
            L.ensure_logits(sh.n_logits)
        rows = dict(f32=self.f32, eps=spec.rms_eps, status=self.status)
        again = dict(tokens=md["tokens"], table=w.embed, scale=spec.embed_scale)
        ops.norm_rows(L.x, spec.hidden, T, xn=L.xn, **again, **rows)
        for k, (freq, amp) in w.rope.items():
            ops.rope_table(md["positions"], freq, amp, L.rope[k], T)
        self.launches_per_step = 1 + len(w.rope)
        for r, (li, _) in enumerate(self.runs):
            b, lw, last = spec.blocks[li], w.layer(li), r + 1 == len(self.runs)
            # what the launch that closes this run leaves for the next one: at the start of a pass behind the first, the embedding output is added before
            opens = {} if last or not self.runs[r + 1][1] else again
            nxt = dict(xn=None if last else L.xn, **({} if self.tap is not None else opens))
            out = L.output(b)
            self._mixer(r, b, lw, L, out, sh)
            if b.ffn is not None:
                self._feed_forward(lw, L, out, T)
            self._dense(lw.wo, out["act"], L.mix, T)
            if spec.side_dim:
                ops.norm_rows(L.x, spec.hidden, T, add=L.mix, xn=L.raw, raw=True, **rows)
                self._dense(lw.side_gate, L.raw_act, L.side_z, T)
                ops.side_gate(L.side_z, md["tokens"], w.side, li * spec.side_dim, spec.side_dim, L.side_g, T, status=self.status)
                self._dense(lw.side_proj, L.side_act, L.mix, T)
                self.launches_per_step += 2
            ops.norm_rows(L.x, spec.hidden, T, add=L.mix, post=lw.side_norm, **nxt, **rows)
            self.launches_per_step += 1
            if self.tap is not None:
                self.tap.append(L.x[:T, :spec.hidden].clone())
                if opens:            # the rows were wanted without the embedding output: it is added on its own
                    ops.norm_rows(L.x, spec.hidden, T, add=torch.zeros_like(L.mix), xn=L.xn, **opens, **rows)
        if sh.n_logits:
            ops.norm_rows(L.x, spec.hidden, sh.n_logits, src_rows=md["logit_rows"], xn=L.xln, **rows)
            ops.tc_linear(w.lm_head, L.head_operand(sh.n_logits), L.logits, rows=sh.n_logits, status=self.status)
            ops.argmax_rows(L.logits, L.next_tok, rows=sh.n_logits, status=L.tok_status)
            self.launches_per_step += 3
        return L

    def _mixer(self, r: int, b: BlockSpec, lw: MixedLayer, L: MixedLane, out: dict, sh: StepShape):
        """Runs a layer run's mixer on L.xn into its columns of the output operand."""
        a, T, m = b.attn, sh.T, L.mixer(b, lw.w_in.N)
        self._dense(lw.w_in, L.xn_act, m["proj"], T)
        if a is None:
            self._hgrn2(r, b.rec, lw, L, m["proj"], out["o"], sh)
        elif a.kind == "latent":
            self._latent(r, a, lw, L, {**m, "o": out["o"]}, sh)
        else:
            extras = ops.attn_extras(pooled=self.pooled.get(r), pool_maps=self.pool_maps.get(r), pool=a.pool) if a.pool else None
            self._attend(r, a, lw, L, m, out["o"], sh, bias=lw.qkv_b, extras=extras, pooled=self.pooled.get(r))

    def _latent(self, r: int, a, lw: MixedLayer, L: MixedLane, m: dict, sh: StepShape):
        T, H, rp, plane = sh.T, a.n_heads, up(a.kv_lora_rank, 64), self.plane[r]
        rope, rows = L.rope[rope_key(a)] if a.rope_dims else None, self.latents[plane]
        ops.latent_down(m["proj"], lw.columns["dq"][0], lw.columns["dkv"][0], lw.q_norm, lw.kv_norm, rope, self.md["slot_map"], m["cq"], rows, T=T, r=a.kv_lora_rank, rp=rp,
                        rot=a.rope_dims, eps=self.spec.rms_eps, status=self.status)
        self._dense(lw.w_uq, m["cq_act"], m["qx"], T)
        ops.latent_split(m["qx"], rope, m["q"], m["qr"], m["tiles"], m["n_tiles"], T=T, ldt=L.cap, H=H, d=a.head_dim, rot=a.rope_dims, tn=L.tn)
        self.launches_per_step += 2
        self._latent_attention(a, lw, L, m, rows, self.kv_tmaps[plane] if self.kv_tmaps is not None else None, None, sh)

    def _hgrn2(self, r: int, spec, lw: MixedLayer, L: MixedLane, proj: torch.Tensor, out: torch.Tensor, sh: StepShape):
        column = lambda name: proj[:, lw.columns[name][0]:]
        state, tags, ring = self.states[r]
        arg = ops.decay_scan_arg(column("rq"), column("rf"), column("rv"), None, state, tags, ring, out, self.md, H=spec.heads, dim=spec.dim, vdim=spec.vdim, n_seq=sh.n_seq,
                                 max_q_len=sh.max_q_len, eps=self.spec.rms_eps, forget=(lw.forget_b, lw.lower), norm=lw.lin_norm, chunks=L.scan_chunks(spec), T=sh.T, status=self.status)
        ops.decay_scan(arg, f32=self.f32)
        self.launches_per_step += 4 if arg.chunks and sh.max_q_len > 16 else 1

    def _feed_forward(self, lw: MixedLayer, L: MixedLane, out: dict, T: int):
        if self.f32:
            self._dense(lw.ws_gate, L.xn_act, out["g"], T)
            self._dense(lw.ws_up, L.xn_act, out["u"], T)
            ops.silu_rows(out["g"], out["u"], out["h"], T)
            self.launches_per_step += 1
        else:
            self._dense(lw.ws_gate, L.xn_glu, out["h"], T, w_up=lw.ws_up)

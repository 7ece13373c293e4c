"""Engine of hybrid recurrent / windowed-attention stacks (the Tudilix design): gated linear recurrences and short-convolution attention over
an fp32 residual, an RMS norm in front of and behind every sub-layer, clamped-GLU feed-forwards.

Runs the generic engine's steps (packed inputs, paged cache, state slots, CUDA graphs per shape, head and token selection) with its own layer
program; every arrow between two products is one launch:

  token row -> x (fp32), h = norm(x)
  attention       h -> queries | keys | values               one product
                  conv_qkv: causal convolution, head norms, rotation -> query rows, paged cache rows, ring of inputs
                  windowed paged attention -> W_o            (layers that share another layer's keys and values project queries only)
  recurrence      h -> y branch | x branch                   one product
                  rglru_conv -> both gates                   one product grouped over the channel blocks, fp32 output
                  lru_scan: gates, recurrence, GELU branch -> W_o
  x += m * norm(mixer), h = norm(x)                          one launch
  feed-forward    h -> clamped GLU (biases and activation in the product's epilogue) -> W_down
  x += m * norm(feed-forward + bias), h = next layer's norm  one launch
  rows that need logits -> final norm -> head (soft cap in its epilogue)

Keys and values live in the paged cache `[layers with keys of their own, slots, row]`.  What a sequence carries besides - convolution inputs,
recurrent states - sits in its state slot, in rings addressed by position: a state slot needs no reset (nothing in front of position 0 is
read), a repeated step repeats its writes, and up to `state_depth` tokens can be taken back by simply continuing from an earlier position, so
drafted tokens need no replay.  With fp32 weights (`QuantSpec.dense = "f32"`) the same program runs entirely in fp32.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config import AttentionSpec, RecurrentSpec
from ..models.hybrid_stack import HybridLayer, HybridWeights, rope_key
from ..models.latent_stack import up
from ..ops import ActBuffer
from .engine import Engine, PAGE, StepShape
from .stack import StackBase, StackLane

SCAN_CHUNK = 64             # tokens of a chunk of the recurrence's long-run form
MAX_TAPS = 16
POOL_ROWS = 16              # runs of up to this many tokens leave the blocks they complete in the launch that writes their keys and values


class HybridLane(StackLane):
    def __init__(self, eng: "HybridStackEngine", cap: int):
        super().__init__(eng, cap)
        # the GLU product pairs two weight tiles: token tiles of at most 128 rows over the same operand rows
        tn = min(self.tn, 128)
        self.xn_glu = self.xn_act if eng.f32 or tn == self.tn else ActBuffer(self.kind, cap, eng.Wp, tn, self.xn, ops.encode_tmap(self.xn, tn))
        self.rope = {k: torch.zeros(cap, f.shape[1], 2, dtype=torch.float32, device=self.dev) for k, (f, _) in (eng.weights.rope or {}).items()}

    def attention(self, a: AttentionSpec, n_in: int) -> dict:
        H, dp, dv, cap = a.n_heads, up(a.head_dim, 64), a.v_head_dim, self.cap

        def make():
            o, o_act = self._operand(cap, up(H * dv, 8))
            return {"proj": torch.zeros(cap, up(n_in, 8), dtype=self.dt, device=self.dev), "q": torch.zeros(cap, H * dp, dtype=self.dt, device=self.dev), "o": o, "o_act": o_act}
        return self.get(("attn", H, a.head_dim, dv, n_in), make)

    def recurrence(self, r: RecurrentSpec) -> dict:
        n8, sq, cap = up(r.width, 8), r.width // r.blocks, self.cap

        def make():
            u, u_act = self._operand(r.blocks * cap, up(sq, 8))
            o, o_act = self._operand(cap, n8)
            per = -(-cap // self.tn)
            f32 = lambda *s: torch.zeros(*s, dtype=torch.float32, device=self.dev)
            return {"proj": torch.zeros(cap, 2 * n8, dtype=self.dt, device=self.dev), "u": u, "u_act": u_act, "gates": f32(cap, 2 * r.width), "o": o, "o_act": o_act,
                    "tiles": torch.zeros(r.blocks * per, 4, dtype=torch.int32, device=self.dev), "n_tiles": torch.zeros(1, dtype=torch.int32, device=self.dev),
                    "agg": f32(cap // SCAN_CHUNK + self.eng.max_seqs + 1, r.width, 2) if cap > SCAN_CHUNK else None}
        return self.get(("rec", r.width, r.blocks), make)

    def ffn(self, width: int) -> dict:
        def make():
            h, h_act = self._operand(self.cap, up(width, 8))
            return {"h": h, "h_act": h_act, **({"g": torch.zeros_like(h), "u": torch.zeros_like(h)} if self.eng.f32 else {})}
        return self.get(("ffn", width), make)


class HybridStackEngine(StackBase, Engine):
    LANE = HybridLane
    state_depth = 8             # tokens of a sequence that can be taken back; the most rows a drafted step may have
    PREFILL_MIN_Q = 64          # query rows of a sequence from which attention takes the 128-key kernel

    def __init__(self, weights: HybridWeights, **kw):
        self._check(weights.spec)
        super().__init__(weights, **kw)

    def _check(self, spec):
        if spec.stack != "hybrid":
            raise ValueError("HybridStackEngine runs hybrid stacks described by ModelSpec.blocks")
        for i, b in enumerate(spec.blocks):
            taps = b.rec.conv_taps if b.rec is not None else b.attn.conv_taps
            if not 1 <= taps <= MAX_TAPS:
                raise ValueError(f"layer {i}: convolutions of 1 to {MAX_TAPS} taps (got {taps})")
            if b.attn is not None and max(b.attn.head_dim, b.attn.v_head_dim) > 256:
                raise ValueError(f"layer {i}: heads of up to 256 dimensions (got {b.attn.head_dim} / {b.attn.v_head_dim})")

    # ------------------------------------------------------------------ cache and state
    def _alloc_attention_state(self):
        from ..utils.memory_ledger import LEDGER
        spec, n, dev = self.spec, self.n_pages * PAGE, self.device
        dt = torch.float32 if self.f32 else torch.bfloat16
        owners = spec.kv_layers()
        # zero-filled: head pads and slots nobody wrote hold finite values
        self.kv = torch.zeros(len(owners), n, max(64, spec.kv_row_elems()), dtype=dt, device=dev)
        self.kv_tmaps = None
        self.plane = {i: owners.index(i if b.attn.kv_from < 0 else b.attn.kv_from) for i, b in enumerate(spec.blocks) if b.attn is not None}
        self.maps = {}
        if not self.f32:
            for i in owners:
                a = spec.blocks[i].attn
                self.maps[self.plane[i]] = ops.encode_window_maps(self.kv[self.plane[i]], a.n_kv_heads, up(a.head_dim, 64), up(a.v_head_dim, 64))
        self.rings = []
        for i in range(spec.n_layers):
            conv = self.weights.layer(i).conv
            self.rings.append(torch.zeros(self.max_seqs, conv.shape[0] - 1 + self.state_depth, conv.shape[1], dtype=dt, device=dev) if conv is not None else None)
        self._alloc_states()
        with LEDGER.scope("kv"):
            LEDGER.charge(sum(t.numel() * t.element_size() for t in self.state_buffers()), "sequence state slots")

    def _alloc_states(self):
        """What the recurrent layers carry per state slot."""
        self.states = [torch.zeros(self.max_seqs, self.state_depth + 1, b.rec.width, dtype=torch.float32, device=self.device) if b.rec is not None else None
                       for b in self.spec.blocks]

    def state_buffers(self) -> list:
        return [t for t in self.rings + self.states if t is not None]

    @staticmethod
    def _visible_pages(a: AttentionSpec, rows: int, max_kv: int = 1 << 40) -> int:
        """Pages a run of `rows` queries can see at most through the layer's window, among kept first keys and pooled blocks of a context of up to
        `max_kv` tokens (a large number without a window)."""
        return min(1 << 20, (a.window + rows - 1 + PAGE - 2) // PAGE + 1 + -(-a.keep_first // PAGE) + (-(-max_kv // (a.pool * PAGE)) if a.pool else 0)) if a.window else 1 << 20

    def attn_splits_for(self, n_seq: int, max_q_len: int, max_kv: int) -> int:
        """The largest split count a layer of the step wants (each takes no more than its window has pages)."""
        if self.f32 or max_q_len > 16:
            return 1
        best = 1
        for b in self.spec.blocks:
            if b.attn is None or b.attn.kind != "conv_gqa":
                continue
            ctas = b.attn.n_kv_heads * n_seq * -(-max_q_len // max(1, 128 // (b.attn.n_heads // b.attn.n_kv_heads)))
            pages = min(max(1, -(-max_kv // PAGE)), self._visible_pages(b.attn, max_q_len, max_kv))
            want = max(1, min(32, 2 * self.sm_count // ctas, pages))
            if want == pages and not (b.attn.window and max_kv > b.attn.window):
                want = 1 << (want.bit_length() - 1)        # a growing context re-captures rarely
            best = max(best, want)
        return best

    # ------------------------------------------------------------------ layer program
    def _forward_single(self, sh: StepShape) -> HybridLane:
        w, spec, T, md, st = self.weights, self.spec, sh.T, self.md, self.status
        L = self.lane(T)
        if sh.n_logits > L.logits.shape[0]:
            L.ensure_logits(sh.n_logits)
        rows = dict(f32=self.f32, eps=spec.rms_eps, status=st)
        ops.norm_rows(L.x, spec.hidden, T, tokens=md["tokens"], table=w.embed, gain=w.layer(0).attn_norm, xn=L.xn, **rows)
        for k, (freq, amp) in w.rope.items():
            ops.rope_table(md["positions"], freq, amp, L.rope[k], T)
        self.launches_per_step = 1 + len(w.rope)
        for li, b in enumerate(spec.blocks):
            lw = w.layer(li)
            if b.rec is not None:
                self._recurrence(li, b.rec, lw, L, sh)
            else:
                self._attention(li, b.attn, lw, L, sh)
            nxt = w.layer(li + 1).attn_norm if li + 1 < spec.n_layers else None
            gain = lw.ffn_norm if b.ffn is not None else nxt
            ops.norm_rows(L.x, spec.hidden, T, add=L.mix, post=lw.attn_post, mult=spec.residual_mult, gain=gain, xn=L.xn if gain is not None else None, **rows)
            if b.ffn is not None:
                self._glu_ffn(b.ffn, lw, L, T)
                ops.norm_rows(L.x, spec.hidden, T, add=L.mix, bias=lw.down_b, post=lw.ffn_post, mult=spec.residual_mult, gain=nxt, xn=L.xn if nxt is not None else None, **rows)
                self.launches_per_step += 1
            self.launches_per_step += 1
            if self.tap is not None:
                self.tap.append(L.x[:T, :spec.hidden].clone())
        if sh.n_logits:
            ops.norm_rows(L.x, spec.hidden, sh.n_logits, src_rows=md["logit_rows"], gain=w.final_norm, xn=L.xln, **rows)
            cap = spec.logit_softcap
            ops.tc_linear(w.lm_head, L.head_operand(sh.n_logits), L.logits, rows=sh.n_logits, act="softcap" if cap else None, bound=cap, status=st)
            ops.argmax_rows(L.logits, L.next_tok, rows=sh.n_logits, status=L.tok_status)
            self.launches_per_step += 3
        return L

    def _attention(self, li: int, a: AttentionSpec, lw: HybridLayer, L: HybridLane, sh: StepShape):
        b = L.attention(a, lw.w_in.N)
        self._dense(lw.w_in, L.xn_act, b["proj"], sh.T)
        self._attend(li, a, lw, L, b, b["o"], sh)
        self._dense(lw.wo, b["o_act"], L.mix, sh.T)

    def _attend(self, li: int, a: AttentionSpec, lw: HybridLayer, L: HybridLane, b: dict, out: torch.Tensor, sh: StepShape, *, bias=None, extras=None, pooled=None):
        """Projected rows b["proj"] -> convolution, norms, rotation, cache (and `pooled` blocks) -> attended rows `out`."""
        T, md, H, G, plane = sh.T, self.md, a.n_heads, a.n_kv_heads, self.plane[li]
        dp, dvp, dv = up(a.head_dim, 64), up(a.v_head_dim, 64), a.v_head_dim
        ops.conv_qkv(b["proj"], lw.conv, lw.q_norm, lw.k_norm, L.rope.get(rope_key(a)), self.rings[li], b["q"], self.kv[plane], md, H=H, G=G if a.kv_from < 0 else 0,
                     dim=a.head_dim, dp=dp, vdim=dv, dvp=dvp, pairs=a.rope_dims // 2, eps=self.spec.rms_eps, n_seq=sh.n_seq, max_q_len=sh.max_q_len, bias=bias,
                     norm="whole" if a.qk_norm_whole else ("head" if a.qk_norm or a.qk_norm_unit else ""), half=not a.rope_interleaved, values_are_keys=a.values_are_keys,
                     n_slots=self.max_seqs, pooled=pooled, pool=a.pool, status=self.status)
        if pooled is not None and sh.max_q_len > POOL_ROWS:
            ops.pool_kv(self.kv[plane], pooled, a.pool, md["page_table"], md["kv_len"], md["q_len"], width=G * (dp + dvp), n_seq=sh.n_seq, max_q_len=sh.max_q_len, status=self.status)
            self.launches_per_step += 1
        where = (md["page_table"], md["kv_len"], md["q_start"], md["q_len"], out)
        shape = dict(T=T, n_seq=sh.n_seq, Hq=H, Hkv=G, dp=dp, dvp=dvp, dv=dv, window=a.window, scale=a.softmax_scale, extras=extras, status=self.status)
        if self.f32 or H // G > 128:
            ops.window_attention_simt(b["q"], self.kv[plane], *where, pool_stride=pooled.stride(0) if pooled is not None else 0, **shape)
        elif sh.max_q_len >= self.PREFILL_MIN_Q and dp + 2 * dvp <= 512:
            ops.window_attention(b["q"], self.maps[plane], *where, max_q_len=sh.max_q_len, prefill=True, **shape)
        else:
            splits = min(sh.attn_splits, self._visible_pages(a, sh.max_q_len))
            if splits > 1:
                self._scratch(splits * T * H * dvp, splits * T * H * 2)
                self.launches_per_step += 1
            ops.window_attention(b["q"], self.maps[plane], *where, max_q_len=sh.max_q_len, n_splits=splits, part_o=self.part_o if splits > 1 else None,
                                 part_ml=self.part_ml if splits > 1 else None, **shape)
        self.launches_per_step += 2

    def _recurrence(self, li: int, r: RecurrentSpec, lw: HybridLayer, L: HybridLane, sh: StepShape):
        T, n8 = sh.T, up(r.width, 8)
        b = L.recurrence(r)
        self._dense(lw.w_in, L.xn_act, b["proj"], T)
        arg = ops.recurrence_arg(b["proj"][:, n8:], b["proj"], lw.x_b, lw.y_b, lw.conv, lw.conv_b, self.rings[li], self.states[li], b["u"], b["gates"], lw.gates_b, lw.decay,
                                 b["agg"], b["o"], self.md, blocks=r.blocks, T=T, ldt=L.cap, tiles=b["tiles"], n_tiles=b["n_tiles"], tn=L.tn, n_seq=sh.n_seq,
                                 max_q_len=sh.max_q_len, status=self.status)
        ops.rglru_conv(arg, f32=self.f32)
        ops.tc_linear(lw.w_gates, b["u_act"], b["gates"], rows=r.blocks * L.cap, tiles=b["tiles"], n_tiles=b["n_tiles"], max_tiles=r.blocks * -(-T // L.tn),
                      token_major=(L.cap, 2 * (r.width // r.blocks)), status=self.status)
        ops.lru_scan(arg, f32=self.f32)
        self._dense(lw.wo, b["o_act"], L.mix, T)
        self.launches_per_step += 3 + (1 if sh.max_q_len > SCAN_CHUNK else 0)

    def _glu_ffn(self, m, lw: HybridLayer, L: HybridLane, T: int):
        b = L.ffn(m.intermediate)
        if self.f32:
            self._dense(lw.ws_gate, L.xn_act, b["g"], T)
            self._dense(lw.ws_up, L.xn_act, b["u"], T)
            ops.glu_rows(b["g"], b["u"], lw.gate_b, lw.up_b, b["h"], T, m.limit)
        else:
            ops.tc_linear(lw.ws_gate, L.xn_glu, b["h"], rows=T, w_up=lw.ws_up, act="clamped_glu", bound=m.limit, biases=(lw.gate_b, lw.up_b), status=self.status)
        self._dense(lw.ws_down, b["h_act"], L.mix, T)
        self.launches_per_step += 1

"""Engine of hyper-connected stacks with side-by-side mixers (the Vozetar design): several fp32 residual streams mixed by constants around every
sub-layer; attention (causal, or windowed with kept first keys) alone or beside a linear mixer (retention, gated linear attention); dense or
routed feed-forwards.

Runs the generic engine's steps (packed inputs, paged cache, state slots, CUDA graphs per shape, head and token selection) with its own layer
program on the hybrid stacks' attention; every arrow between two products is one launch:

  token row + pair row -> every stream, h = norm(collapsed streams)
  mixer          h -> queries | keys | values | gate | linear mixer's queries, keys, values, gate, decay input       one product
                 conv_qkv: bias, convolution, norm, rotation -> query rows, paged cache rows, ring of inputs
                 paged attention (window, kept first keys, sink, gate) -> columns of the output operand
                 decay_scan: rotation, decays, recurrence, output norm, gate -> the columns behind them (prompts: four launches, in chunks)
                 -> W_o          (one product over both, or one each where the outputs are normalised before they are added)
  streams <- constants x (streams, mixer), h = norm(collapsed streams)                                               one launch
  feed-forward   h -> SwiGLU in the product's epilogue -> W_down;  routed: router -> selection + packing -> gather -> grouped products
  streams <- constants x (streams, feed-forward [+ weighted routed rows]), h = next layer's                          one launch
  rows that need logits: sum of the streams -> final norm -> head

Keys and values live in the paged cache like the hybrid stacks'.  What a sequence carries besides sits in its state slot: convolution inputs and
fed tokens in rings addressed by position, the linear mixers' states in two places tagged with their positions (see `csrc/decay_scan.cu`).  A
slot needs no reset, a repeated step repeats its writes, and up to `state_depth` tokens can be taken back by continuing from an earlier
position.  With fp32 weights (`QuantSpec.dense = "f32"`) the same program runs entirely in fp32.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config import BlockSpec, MoESpec, RecurrentSpec
from ..models.hybrid_stack import rope_key
from ..models.hyper_stack import HyperLayer, check_blocks
from ..models.latent_stack import up
from .engine import StepShape
from .hybrid_stack import HybridLane, HybridStackEngine

ROUTER_ROWS = 64            # steps of up to this many rows take the router's logits from the ordinary cores


class HyperLane(HybridLane):
    def __init__(self, eng: "HyperStackEngine", cap: int):
        super().__init__(eng, cap)
        self.mix2 = torch.zeros_like(self.mix) if any(b.merge_norm for b in eng.spec.blocks) else None

    def mixer(self, b: BlockSpec, n_in: int) -> dict:
        """Buffers of one mixer geometry: projection rows, query rows, and the output projection's operand(s) - attention's columns first."""
        a, r, cap = b.attn, b.rec, self.cap
        K1, K2 = up(a.n_heads * a.v_head_dim, 8), up(r.heads * r.vdim, 8) if r is not None else 0

        def make():
            d = {"proj": torch.zeros(cap, up(n_in, 8), dtype=self.dt, device=self.dev), "q": torch.zeros(cap, a.n_heads * up(a.head_dim, 64), dtype=self.dt, device=self.dev)}
            o, d["o_act"] = self._operand(cap, K1 if b.merge_norm else K1 + K2)
            d["o"], d["r"] = o[:, :K1], o[:, K1:]
            if b.merge_norm:
                d["r"], d["r_act"] = self._operand(cap, K2)
            return d
        return self.get(("mix", a.n_heads, a.head_dim, a.v_head_dim, K2, b.merge_norm, n_in), make)


    def scan_chunks(self, r: RecurrentSpec) -> tuple | None:
        """Scratch of a linear mixer's long runs (none in the all-fp32 mode, for decode-sized lanes and for heads the chunk kernels do not take)."""
        if self.eng.f32 or self.cap <= 16 or r.dim > 128 or r.vdim > 256:
            return None
        return self.get(("scan", r.heads, r.dim, r.vdim), lambda: ops.scan_scratch(self.cap, self.eng.max_seqs, r.heads, r.dim, r.vdim, self.dev))


class HyperStackEngine(HybridStackEngine):
    LANE = HyperLane

    def _check(self, spec):
        if spec.stack != "hyper":
            raise ValueError("HyperStackEngine runs hyper-connected stacks described by ModelSpec.blocks and ModelSpec.streams")
        check_blocks(spec)

    @property
    def residual_shape(self) -> tuple:
        return (self.spec.streams, self.Wp)

    # ------------------------------------------------------------------ state
    def _alloc_states(self):
        n, D, dev = self.max_seqs, self.state_depth, self.device
        f32 = lambda *s: torch.zeros(*s, dtype=torch.float32, device=dev)
        self.states = []            # per layer: (two states per head, their positions, inputs of the last tokens)
        for b in self.spec.blocks:
            r = b.rec
            vp = up(r.vdim, 4) if r is not None else 0
            self.states.append((f32(n, 2, r.heads, r.dim, vp), torch.zeros(n, r.heads, 2, dtype=torch.int32, device=dev), f32(n, D, r.heads, 2 * r.dim + vp))
                               if r is not None else None)
        self.recent = torch.zeros(n, D + 1, dtype=torch.int32, device=dev)       # tokens by position

    def state_buffers(self) -> list:
        return [t for t in self.rings if t is not None] + [t for s in self.states if s is not None for t in s] + [self.recent]

    # ------------------------------------------------------------------ layer program
    def _forward_single(self, sh: StepShape) -> HyperLane:
        w, spec, T, md = self.weights, self.spec, sh.T, self.md
        L = self.lane(T)
        if sh.n_logits > L.logits.shape[0]:
            L.ensure_logits(sh.n_logits)
        rows = dict(f32=self.f32, eps=spec.rms_eps, status=self.status)
        opens = [(lw.hc1[0], lw.attn_norm) for lw in (w.layer(i) for i in range(spec.n_layers))] + [None]

        def reads(nxt):
            """The next sub-layer's stream weights and norm, for the launch that leaves its input (nothing behind the last one)."""
            return dict(next_in=nxt[0], gain=nxt[1], xn=L.xn) if nxt is not None else {}

        pt = spec.pair_table
        ops.hyper_rows(L.x, spec.hidden, T, tokens=md["tokens"], table=w.embed, pairs=(w.pair_rows, pt.mul_prev, pt.mul_cur, self.recent) if pt is not None else None,
                       meta=md, n_seq=sh.n_seq, **reads(opens[0]), **rows)
        for k, (freq, amp) in w.rope.items():
            ops.rope_table(md["positions"], freq, amp, L.rope[k], T)
        self.launches_per_step = 1 + len(w.rope)
        for li, b in enumerate(spec.blocks):
            lw = w.layer(li)
            ffn = b.ffn is not None or b.moe is not None
            y = self._mixer(li, b, lw, L, sh)
            ops.hyper_rows(L.x, spec.hidden, T, out=lw.hc1[1], mix=lw.hc1[2], **y, **reads((lw.hc2[0], lw.ffn_norm) if ffn else opens[li + 1]), **rows)
            if ffn:
                y = self._feed_forward(b, lw, L, T)
                ops.hyper_rows(L.x, spec.hidden, T, out=lw.hc2[1], mix=lw.hc2[2], **y, **reads(opens[li + 1]), **rows)
                self.launches_per_step += 1
            self.launches_per_step += 1
            if self.tap is not None:
                self.tap.append(L.x[:T, :, :spec.hidden].sum(1))
        if sh.n_logits:
            ops.hyper_rows(L.x, spec.hidden, sh.n_logits, src_rows=md["logit_rows"], gain=w.final_norm, xn=L.xln, **rows)
            ops.tc_linear(w.lm_head, L.head_operand(sh.n_logits), L.logits, rows=sh.n_logits, status=self.status)
            ops.argmax_rows(L.logits, L.next_tok, rows=sh.n_logits, status=L.tok_status)
            self.launches_per_step += 3
        return L

    def _mixer(self, li: int, b: BlockSpec, lw: HyperLayer, L: HyperLane, sh: StepShape) -> dict:
        """Runs a layer's mixer(s) on L.xn; returns what the stream boundary adds."""
        T, a, r = sh.T, b.attn, b.rec
        m = L.mixer(b, lw.w_in.N)
        self._dense(lw.w_in, L.xn_act, m["proj"], T)
        column = lambda name: m["proj"][:, lw.columns[name][0]:]
        merged = r is not None and not b.merge_norm
        extras = ops.attn_extras(sink=lw.sink, gate=column("gate") if a.out_gate else None, per_value=a.gate_values, keep_first=a.keep_first,
                                 out_scale=b.merge_scales[0] if merged else 1.0)
        self._attend(li, a, lw, L, m, m["o"], sh, bias=lw.qkv_b, extras=extras)
        if r is not None:
            state, tags, ring = self.states[li]
            gla = r.kind == "gla"
            arg = ops.decay_scan_arg(column("rq"), column("rk"), column("rv"), column("rg"), state, tags, ring, m["r"], self.md, H=r.heads, dim=r.dim, vdim=r.vdim,
                                     n_seq=sh.n_seq, max_q_len=sh.max_q_len, eps=self.spec.rms_eps, rope=L.rope[rope_key(r)] if r.rope_dims else None,
                                     pairs=r.rope_dims // 2, q_scale=r.dim ** -0.5 if gla else 1.0, k_scale=1.0 if gla else r.dim ** -0.5, decay=lw.lin_decay,
                                     low_rank=(column("a1"), lw.lin_a2, lw.lin_a2_b) if gla else None, tau=r.tau, norm=lw.lin_norm,
                                     out_scale=b.merge_scales[1] if merged else 1.0, chunks=L.scan_chunks(r), T=T, status=self.status)
            ops.decay_scan(arg, f32=self.f32)
            self.launches_per_step += 4 if arg.chunks and sh.max_q_len > 16 else 1
        self._dense(lw.wo, m["o_act"], L.mix, T)
        if not b.merge_norm:
            return dict(a=L.mix, bias=lw.wo_b)
        self._dense(lw.wo2, m["r_act"], L.mix2, T)
        return dict(a=L.mix, b=L.mix2, norms=lw.merge_norms, scales=b.merge_scales)

    def _feed_forward(self, b: BlockSpec, lw: HyperLayer, L: HyperLane, T: int) -> dict:
        m = b.moe
        if m is None:
            self._silu_ffn(b.ffn.intermediate, lw, L, T)
            return dict(a=L.mix)
        e = L.experts(m)
        self._router_logits(m, lw, L, e, T)
        self._experts(m, lw, L, e, T)
        if m.n_shared:
            self._silu_ffn(m.shared_inter, lw, L, T)
        return dict(a=L.mix if m.n_shared else None, routed=(e["y"], e["slot"], e["wts"], m.top_k))

    def _router_logits(self, m: MoESpec, lw: HyperLayer, L: HyperLane, e: dict, T: int):
        if not self.f32 and T <= ROUTER_ROWS:
            ops.router_logits(L.xn, lw.router, e["logits"], T)
            self.launches_per_step += 1
        else:
            self._dense(lw.router, L.xn_glu, e["logits"], T)      # (narrow products spread better over 128-row tiles)

    def _silu_ffn(self, width: int, lw: HyperLayer, L: HyperLane, T: int):
        """Dense feed-forward or shared expert: L.xn -> L.mix."""
        b = L.ffn(width)
        if self.f32:
            self._dense(lw.ws_gate, L.xn_act, b["g"], T)
            self._dense(lw.ws_up, L.xn_act, b["u"], T)
            ops.silu_rows(b["g"], b["u"], b["h"], T)
            self.launches_per_step += 1
        else:
            self._dense(lw.ws_gate, L.xn_glu, b["h"], T, w_up=lw.ws_up)
        self._dense(lw.ws_down, b["h_act"], L.mix, T)

"""What the engines of layer stacks share: a lane over fp32 residual rows, bf16 or fp32 operands, lanes of prompt size, lazily made buffers, routed
experts."""
from __future__ import annotations

import math
import os

import torch

from .. import ops
from ..models.latent_stack import up
from ..ops import ActBuffer, KIND_BF16, KIND_F32, pick_tn
from ..ops.native import call, ptr, stream
from .engine import Lane

LANE_CAPS = (16, 32, 64, 256, 1024, 4096, 16384)
NARROW_WEIGHTS = 36 << 20       # most weights of a product that 33 to 64 rows take in tiles of 32 (a cluster splits K; wider ones read their weights once)


class StackLane(Lane):
    """Activation buffers for steps of up to `cap` rows; buffers that depend on a layer's geometry are made on first use per geometry."""

    def __init__(self, eng: "StackBase", cap: int):
        self.eng, self.cap, self.dev = eng, cap, eng.device
        self.dt = torch.float32 if eng.f32 else torch.bfloat16
        self.kind = KIND_F32 if eng.f32 else KIND_BF16
        # products of one weight tile keep both accumulators with 256-row token tiles: prompt-sized lanes take them
        self.tn = pick_tn(min(cap, int(os.environ.get("CUTEAFD_TN", "256" if cap >= 1024 else "128"))))
        Wp = eng.Wp
        self.x = torch.zeros(cap, *eng.residual_shape, dtype=torch.float32, device=self.dev)
        self.xn, self.xn_act = self._operand(cap, Wp)
        self.mix = torch.zeros(cap, Wp, dtype=self.dt, device=self.dev)
        rows = min(cap, 256)
        self.xln, self.xln_act = self._operand(rows, Wp)
        self._head_acts: dict = {}
        self.logits = torch.zeros(rows, eng.spec.vocab, dtype=torch.float32, device=self.dev)
        i32 = lambda *s: torch.zeros(*s, dtype=torch.int32, device=self.dev)
        self.next_tok, self.tok_status = i32(cap), i32(cap)
        self._bufs: dict = {}

    def _operand(self, rows: int, K: int, tn: int | None = None):
        act = ActBuffer.alloc(self.kind, rows, K, tn or self.tn, self.dev)
        return act.data, act

    def ensure_logits(self, n: int):
        """Steps that want more logit rows than a lane starts with (whole prompts scored position by position)."""
        if n > self.logits.shape[0]:
            rows = min(self.cap, up(n, 256))
            self.xln, self.xln_act = self._operand(rows, self.eng.Wp)
            self.logits = torch.zeros(rows, self.eng.spec.vocab, dtype=torch.float32, device=self.dev)
            self._head_acts.clear()
            self.eng.drop_graphs()                   # captured steps hold the old addresses

    def retiled(self, act: ActBuffer, tn: int) -> ActBuffer:
        """The same operand rows in token tiles of `tn` (made in the eager run of a new shape)."""
        if tn == act.tn or act.kind != KIND_BF16:
            return act
        return self.get(("tiles", act.data.data_ptr(), act.K, tn), lambda: ActBuffer(act.kind, act.rows, act.K, tn, act.data, ops.encode_tmap(act.data, tn)))

    def head_operand(self, n: int) -> ActBuffer:
        """The head's operand in token tiles that fit the `n` rows it multiplies (a prompt's step has few)."""
        tn = pick_tn(min(n, self.tn))
        if self.eng.f32 or tn == self.xln_act.tn:
            return self.xln_act
        if tn not in self._head_acts:
            self._head_acts[tn] = ActBuffer(self.kind, self.xln.shape[0], self.eng.Wp, tn, self.xln, ops.encode_tmap(self.xln, tn))
        return self._head_acts[tn]

    def experts(self, m) -> dict:
        E, k, ff, cap = m.n_experts, m.top_k, m.intermediate, self.cap
        glu = m.activation == "swiglu"

        def make():
            rows = cap * k
            # rows per expert of a full lane: whole 256-row tiles where they fill, else about twice the mean (a product of two weight tiles
            # takes at most 128)
            mean = max(1, math.ceil(rows / E))
            tn = pick_tn(min(mean if mean >= 256 else min(2 * mean, 128), int(os.environ.get("CUTEAFD_TNG", "256"))), swiglu=glu)
            i32 = lambda *s: torch.zeros(*s, dtype=torch.int32, device=self.dev)
            xs, xs_act = self._operand(rows, self.eng.Wp, tn)
            h1, h1_act = self._operand(rows, up(ff, 8), tn)
            max_tiles = E + rows // tn + 1
            return {"tn": tn, "max_tiles": max_tiles, "logits": torch.zeros(cap, E, dtype=torch.float32, device=self.dev), "idx": i32(cap, k),
                    "wts": torch.zeros(cap, k, dtype=torch.float32, device=self.dev), "src": i32(rows), "slot": i32(cap, k), "counts": i32(E),
                    "offsets": i32(E), "tiles": i32(max_tiles, 4), "n_tiles": i32(1), "n_rows": i32(1), "xs": xs, "xs_act": xs_act, "h1": h1,
                    "h1_act": h1_act, "y": torch.zeros(rows, self.eng.Wp, dtype=self.dt, device=self.dev),
                    **({"g": torch.zeros_like(h1), "u": torch.zeros_like(h1)} if glu and self.eng.f32 else {})}
        return self.get(("moe", E, k, ff, m.activation), make)

    def latent(self, H: int, rp: int) -> dict:
        """Operands of the absorbed form: query and attended rows in the latent space."""
        def make():
            q, _ = self._operand(H * self.cap, rp)
            o, o_act = self._operand(H * self.cap, rp)
            return {"q": q, "o": o, "o_act": o_act}
        return self.get(("lat", H, rp), make)

    def get(self, key, make):
        if key not in self._bufs:
            self._bufs[key] = make()
        return self._bufs[key]


class StackBase:
    """Mixed in front of an engine class; `LANE` is its lane class."""
    LANE = StackLane

    def __init__(self, weights, **kw):
        self.f32, self.Wp = weights.f32, up(weights.spec.hidden, 8)
        self.tap = None             # set to a list to collect the residual rows after every layer run of eager steps
        super().__init__(weights, **kw)

    @property
    def residual_shape(self) -> tuple:
        """Shape of a token's residual rows."""
        return (self.Wp,)

    def lane(self, T: int) -> StackLane:
        cap = next(c for c in LANE_CAPS if T <= c)
        if cap not in self.lanes:
            self.lanes[cap] = self.LANE(self, cap)
        return self.lanes[cap]

    def drop_graphs(self):
        self.graphs.clear()
        self.census.invalidate()

    def cache_buffers(self) -> list:
        """What the paged cache consists of."""
        return [self.kv]

    def _scratch(self, n_o: int, n_ml: int):
        """Partial outputs and (max, sum) pairs of split attention: grows to the largest need of any layer, in the eager run of a new shape."""
        o, ml = (t.numel() if t is not None else 0 for t in (getattr(self, "part_o", None), getattr(self, "part_ml", None)))
        if o < n_o or ml < n_ml:
            if o:
                self.drop_graphs()                         # captured steps hold the old scratch
            self.part_o = torch.empty(max(o, n_o), dtype=torch.float32, device=self.device)
            self.part_ml = torch.empty(max(ml, n_ml), dtype=torch.float32, device=self.device)

    def set_input_embeds(self, rows, vals):
        if vals is not None and len(rows):
            raise NotImplementedError("image / audio rows are not wired for layer stacks")

    def _dense(self, w, x_act, y, T, residual=None, w_up=None):
        """Products that leave most of the machine idle take smaller token tiles than their lane's: of 32 rows, whose clusters split K, in small steps;
        in prompts as small as it takes for every SM to have one."""
        if w_up is None and w.kind == KIND_BF16:
            tn, nt = x_act.tn, -(-w.N // 128)
            if 32 < T <= 64 and w.N * w.K <= NARROW_WEIGHTS and 4 * nt <= self.sm_count:
                tn = 32
            elif T >= 1024:
                while tn > 32 and nt * -(-T // tn) < self.sm_count:
                    tn //= 2
            x_act = self.lane(T).retiled(x_act, tn)
        super()._dense(w, x_act, y, T, residual=residual, w_up=w_up)

    def _splits(self, N, K, T, tn, kind):
        """Short tiles of 64 rows gain from the fix-up of a split only while they leave three of four SMs idle (measured on B200)."""
        if kind == KIND_F32 or (kind == KIND_BF16 and tn == 64 and T <= 64 and K <= 8192 and 4 * -(-N // 128) > self.sm_count):
            return 1
        return super()._splits(N, K, T, tn, kind)

    def _experts(self, m, lw, L: StackLane, e: dict, T: int):
        """Routing, packing, gather and the experts' products of the rows L.xn, from router logits in e["logits"]: weighted rows stay in e."""
        E, k = m.n_experts, m.top_k
        sel = (e["logits"], None, e["idx"], e["wts"], T, k, m.scoring, m.normalize, m.route_scale, m.n_group, m.topk_group)
        if T * k <= 1024:
            ops.router_select_pack(*sel, e["src"], e["slot"], e["counts"], e["offsets"], e["tiles"], e["n_tiles"], e["n_rows"], 0, E, e["tn"], e["max_tiles"],
                                   group_score=m.group_score)
        else:
            ops.router_select(*sel, group_score=m.group_score)
            ops.route_pack(e["idx"], e["src"], e["slot"], e["counts"], e["offsets"], e["tiles"], e["n_tiles"], e["n_rows"], T, k, 0, E, e["tn"], e["max_tiles"])
            self.launches_per_step += 1
        rows = T * k
        call("cuteafd_gather_rows", ptr(L.xn), ptr(e["src"]), ptr(e["n_rows"]), ptr(e["xs"]), rows, self.Wp * L.xn.element_size() // 2, stream())
        tiles = dict(tiles=e["tiles"], n_tiles=e["n_tiles"], max_tiles=min(e["max_tiles"], E + rows // e["tn"] + 1), status=self.status)
        if m.activation == "relu2":
            ops.tc_linear(lw.w_up, e["xs_act"], e["h1"], rows=rows, act="relu2", **tiles)
        elif self.f32:
            ops.tc_linear(lw.w_gate, e["xs_act"], e["g"], rows=rows, **tiles)
            ops.tc_linear(lw.w_up, e["xs_act"], e["u"], rows=rows, **tiles)
            ops.silu_rows(e["g"], e["u"], e["h1"], rows)
        else:
            ops.tc_linear(lw.w_gate, e["xs_act"], e["h1"], rows=rows, w_up=lw.w_up, **tiles)
        ops.tc_linear(lw.w_down, e["h1_act"], e["y"], rows=rows, **tiles)
        self.launches_per_step += 4

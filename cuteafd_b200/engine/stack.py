"""What the engines of layer stacks share: a lane over fp32 residual rows, bf16 or fp32 operands, lanes of prompt size, lazily made buffers."""
from __future__ import annotations

import os

import torch

from .. import ops
from ..models.latent_stack import up
from ..ops import ActBuffer, KIND_BF16, KIND_F32, pick_tn
from .engine import Lane

LANE_CAPS = (16, 32, 64, 256, 1024, 4096, 16384)


class StackLane(Lane):
    """Activation buffers for steps of up to `cap` rows; buffers that depend on a layer's geometry are made on first use per geometry."""

    def __init__(self, eng: "StackBase", cap: int):
        self.eng, self.cap, self.dev = eng, cap, eng.device
        self.dt = torch.float32 if eng.f32 else torch.bfloat16
        self.kind = KIND_F32 if eng.f32 else KIND_BF16
        # products of one weight tile keep both accumulators with 256-row token tiles: prompt-sized lanes take them
        self.tn = pick_tn(min(cap, int(os.environ.get("CUTEAFD_TN", "256" if cap >= 1024 else "128"))))
        Wp = eng.Wp
        self.x = torch.zeros(cap, Wp, dtype=torch.float32, device=self.dev)
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

    def head_operand(self, n: int) -> ActBuffer:
        """The head's operand in token tiles that fit the `n` rows it multiplies (a prompt's step has few)."""
        tn = pick_tn(min(n, self.tn))
        if self.eng.f32 or tn == self.xln_act.tn:
            return self.xln_act
        if tn not in self._head_acts:
            self._head_acts[tn] = ActBuffer(self.kind, self.xln.shape[0], self.eng.Wp, tn, self.xln, ops.encode_tmap(self.xln, tn))
        return self._head_acts[tn]

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

    def lane(self, T: int) -> StackLane:
        cap = next(c for c in LANE_CAPS if T <= c)
        if cap not in self.lanes:
            self.lanes[cap] = self.LANE(self, cap)
        return self.lanes[cap]

    def drop_graphs(self):
        self.graphs.clear()
        self.census.invalidate()

    def set_input_embeds(self, rows, vals):
        if vals is not None and len(rows):
            raise NotImplementedError("image / audio rows are not wired for layer stacks")

    def _splits(self, N, K, T, tn, kind):
        return 1 if kind == KIND_F32 else super()._splits(N, K, T, tn, kind)

"""Tensor-level wrappers over the native sm_100a kernels.

Each function validates shapes/dtypes, then launches on the current CUDA stream (so callers can capture
whole steps into CUDA graphs).  Nothing here falls back to PyTorch math on a GPU: if the native library is
missing the call raises.  The fp32 oracles live in `cuteafd_b200.ref`.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import native
from .native import call, ptr, stream

KIND_BF16, KIND_NVFP4, KIND_MXFP4, KIND_FP8B = 0, 1, 2, 3      # FP8B: E4M3 with fp32 scales per 128 x 128 (weights) / 1 x 128 (activations)
KIND_W4A8 = 4      # MXFP4 weights x FP8 E4M3 activations, UE8M0 scales per 32 on both (tcgen05 kind::mxf8f6f4)
KIND_F32 = 5       # plain fp32 operands (csrc/f32_linear.cu): the all-fp32 mode of an engine
# MXFP4 expert weights run with MXFP4 activations (W4A4) unless CUTEAFD_MXFP4_ACT=fp8 selects FP8 activations (W4A8, the
# reference's default expert arithmetic; also reachable per model as the "mxfp4_w4a8" format name)
import os as _os
MXFP4_ACT = _os.environ.get("CUTEAFD_MXFP4_ACT", "fp4")
KIND_BY_NAME = {"bf16": KIND_BF16, "nvfp4": KIND_NVFP4, "mxfp4": KIND_W4A8 if MXFP4_ACT == "fp8" else KIND_MXFP4, "mxfp4_w4a4": KIND_MXFP4,
                "mxfp4_w4a8": KIND_W4A8, "fp8_block128": KIND_FP8B, "f32": KIND_F32}
FP4_KINDS = (KIND_NVFP4, KIND_MXFP4)
# activation formats the norm kernels (add_rmsnorm, moe_combine with the next layer's norm) can write in the same launch, and the
# code the native side knows them by
FUSED_QUANT_KINDS = (KIND_NVFP4, KIND_MXFP4, KIND_FP8B)
_QKIND = {KIND_NVFP4: 1, KIND_MXFP4: 2, KIND_FP8B: 3}
EPI_BF16, EPI_BF16_RESIDUAL, EPI_F32 = 0, 1, 3
SCORING = {"sigmoid": 0, "softmax": 1, "sqrtsoftplus": 2}
ACTIVATIONS = {None: 0, "relu2": 1, "softcap": 2, "clamped_glu": 3}      # of a product's epilogue
GROUP_BY_MAX = 16      # added to the scoring code: a group of experts is ranked by its best member (default: the sum of its two best)


def _chk(t: torch.Tensor, dtype, name: str):
    if t.dtype != dtype or not t.is_cuda or not t.is_contiguous():
        raise ValueError(f"{name}: expected contiguous CUDA {dtype}, got {t.dtype} cuda={t.is_cuda} contiguous={t.is_contiguous()}")


# ------------------------------------------------------------------ launch mode / tracing
def set_pdl(mask: int) -> None:
    """Programmatic dependent launch per kernel class (bit 0 glue kernels, bit 1 GEMMs, bit 2 attention; 0 = off, the
    default; CUTEAFD_PDL=<mask> sets it from the environment).  Graphs captured earlier keep their mode."""
    native.lib().cuteafd_set_pdl(int(mask))


_CLUSTER_CAP: dict = {}


def cluster_capacity(kind: int, tn: int, splits: int) -> int:
    """Clusters of `splits` CTAs of the cluster split-K GEMM that fit the device at once (cached per device)."""
    key = (torch.cuda.current_device(), kind, tn, splits)
    if key not in _CLUSTER_CAP:
        out = ctypes.c_int(0)
        call("cuteafd_tc_cluster_capacity", kind, tn, splits, ctypes.addressof(out))
        _CLUSTER_CAP[key] = out.value
    return _CLUSTER_CAP[key]


def fp8_cluster_capacity(tn: int, splits: int, K: int) -> int:
    """Clusters of `splits` CTAs of the FP8 block-scaled GEMM that fit the device at once for this K (cached per device)."""
    key = (torch.cuda.current_device(), "fp8", tn, splits, K)
    if key not in _CLUSTER_CAP:
        out = ctypes.c_int(0)
        call("cuteafd_fp8_cluster_capacity", tn, splits, K, ctypes.addressof(out))
        _CLUSTER_CAP[key] = out.value
    return _CLUSTER_CAP[key]


def tc_trace(buf: torch.Tensor | None, units: int = 0) -> None:
    """Per-unit device time stamps of later `tc_linear` launches: int64 [grid, units, 8] (None = off).  `units < 0`: the cluster
    split-K kernel records instead - its launches with N == -units write eight global-timer stamps per CTA into int64 [grid, 8]
    (entry, -, released by the previous kernel, first stage landed, last MMA committed, accumulator complete, cluster barrier
    passed, epilogue done); usable inside a replayed step graph, where the last such launch of the step survives."""
    call("cuteafd_tc_trace", ptr(buf), units)


# ------------------------------------------------------------------ TMA descriptors
def encode_tmap(t: torch.Tensor, box_rows: int, unpack4: bool = False) -> torch.Tensor:
    """Descriptor array (uint8 [G, 128], on t's device) for a K-major operand [G, rows, K] or [rows, K].
    bf16 tensors describe K elements; uint8 tensors describe K bytes (packed fp4 / fp8).  `unpack4`: a uint8 tensor of packed
    4-bit elements whose tiles TMA expands into 8-bit containers in shared memory (the weight operand of the W4A8 kind)."""
    if t.dim() == 2:
        t = t.unsqueeze(0)
    G, rows, kdim = t.shape
    eb = {torch.bfloat16: 2, torch.uint8: 1}[t.dtype]
    if t.stride(2) != 1:
        raise ValueError("operand must be K-contiguous")
    host = torch.zeros(G, 128, dtype=torch.uint8)
    for g in range(G):
        if unpack4:
            call("cuteafd_tmap_encode_kmajor", host[g].data_ptr(), t[g].data_ptr(), 0, kdim * 2, rows, 1, t.stride(1), 0, box_rows)
        else:
            call("cuteafd_tmap_encode_kmajor", host[g].data_ptr(), t[g].data_ptr(), eb, kdim, rows, 1,
                 t.stride(1) * eb, 0, box_rows)
    return host.to(t.device)


def swizzle_sf(sf: torch.Tensor, per_stage: int = 4) -> torch.Tensor:
    """[rows, n_sf] uint8 block scales -> flat 128x4-atom layout (any device); see ref.quant.swizzle_sf_128x4.
    The scale count per row is zero-padded to whole pipeline stages (`per_stage` scales: 16 NVFP4, 8 MXFP4)."""
    rows, n = sf.shape
    R, Cc = -(-rows // 128) * 128, -(-n // per_stage) * per_stage
    pad = sf.new_zeros(R, Cc)
    pad[:rows, :n] = sf
    return pad.reshape(R // 128, 4, 32, Cc // 4, 4).permute(0, 3, 2, 1, 4).contiguous().reshape(-1)


@dataclass
class TcWeight:
    """Weight set for `tc_linear`: G matrices [N, K] (G > 1 = experts), K-major as checkpoints ship them."""
    kind: int
    G: int
    N: int
    K: int
    data: torch.Tensor              # bf16 [G, N, K] | uint8 [G, N, K/2]
    tmap: torch.Tensor              # uint8 [G, 128]
    sf: torch.Tensor | None = None  # uint8 [G, swizzled bytes]
    sf_ptrs: torch.Tensor | None = None
    alpha: torch.Tensor | None = None   # fp32 [G]: weight global scale x activation global scale (bf16, fp32: an output factor)
    inv_act_gs: torch.Tensor | None = None  # fp32 [1]: 1 / activation global scale (NVFP4)

    @property
    def nbytes(self) -> int:
        return self.data.numel() * self.data.element_size() + (self.sf.numel() if self.sf is not None else 0)

    @staticmethod
    def from_master(w: torch.Tensor, kind: str | int, device, act_gs: float = 1.0 / 64) -> "TcWeight":
        """Quantise fp32 masters [G, N, K] (or [N, K]) with the CPU oracle and upload (tests, small models)."""
        from ..ref import quant
        kind = KIND_BY_NAME[kind] if isinstance(kind, str) else kind
        if w.dim() == 2:
            w = w.unsqueeze(0)
        G, N, K = w.shape
        if kind == KIND_BF16:
            data = w.to(torch.bfloat16).to(device).contiguous()
            return TcWeight(kind, G, N, K, data, encode_tmap(data, 128))
        if kind == KIND_F32:
            return TcWeight(kind, G, N, K, w.to(torch.float32).to(device).contiguous(), None)
        if kind == KIND_FP8B:
            qs = [quant.fp8_block_quantize(w[g]) for g in range(G)]
            data = torch.stack([q for q, _ in qs]).to(device).contiguous()
            return TcWeight(kind, G, N, K, data, encode_tmap(data, 128), torch.stack([s for _, s in qs]).to(device).contiguous())
        packs, sfs, alphas = [], [], []
        for g in range(G):
            if kind == KIND_NVFP4:
                p, s, gs = quant.nvfp4_quantize(w[g])
                alphas.append(float(gs) * act_gs)
            else:
                p, s = quant.mxfp4_quantize(w[g])
                alphas.append(1.0)
            packs.append(p)
            sfs.append(swizzle_sf(s, SF_PER_STAGE[kind]))
        data = torch.stack(packs).to(device).contiguous()
        sf = torch.stack(sfs).to(device).contiguous()
        return TcWeight._finish(kind, G, N, K, data, sf, torch.tensor(alphas, dtype=torch.float32, device=device), act_gs)

    @staticmethod
    def fuse_rows_fp8(a: "TcWeight", b: "TcWeight") -> "TcWeight":
        """One FP8 block-scaled weight [N_a + N_b, K] out of two with the same K (gate and up projections read the same operand:
        one GEMM instead of two).  `a` and `b` become views into the fused storage, so nothing is held twice."""
        if a.kind != KIND_FP8B or b.kind != KIND_FP8B or a.G != 1 or b.G != 1 or a.K != b.K or a.N % 128 or b.N % 128:
            raise ValueError("fuse_rows_fp8: two dense FP8 weights with the same K and row counts that are multiples of 128")
        data = torch.cat([a.data, b.data], 1).contiguous()
        sf = torch.cat([a.sf, b.sf], 1).contiguous()
        fused = TcWeight(KIND_FP8B, 1, a.N + b.N, a.K, data, encode_tmap(data, 128), sf)
        na, ra = a.N, a.N // 128
        a.data, a.sf = data[:, :na], sf[:, :ra]
        b.data, b.sf = data[:, na:], sf[:, ra:]
        a.tmap, b.tmap = encode_tmap(a.data, 128), encode_tmap(b.data, 128)
        return fused

    @staticmethod
    def random(G: int, N: int, K: int, kind: str | int, device, std: float = 0.02, act_gs: float = 1.0 / 64,
               seed: int = 0, groups: tuple | None = None) -> "TcWeight":
        """Random-init weights generated directly in the storage format on the device (large synthetic models).
        `groups=(lo, hi)` keeps only groups [lo, hi) of the G generated ones, so an expert-parallel rank holds exactly
        the experts a single-GPU model of the same seed has at those indices."""
        kind = KIND_BY_NAME[kind] if isinstance(kind, str) else kind
        gen = torch.Generator(device=device).manual_seed(seed)
        lo, hi = groups if groups is not None else (0, G)
        cut = (lambda t: t[lo:hi].clone()) if (lo, hi) != (0, G) else (lambda t: t)
        if kind == KIND_F32:
            return TcWeight(kind, hi - lo, N, K, cut(torch.empty(G, N, K, dtype=torch.float32, device=device).normal_(0, std, generator=gen)), None)
        if kind == KIND_BF16:
            data = cut(torch.empty(G, N, K, dtype=torch.bfloat16, device=device).normal_(0, std, generator=gen))
            return TcWeight(kind, hi - lo, N, K, data, encode_tmap(data, 128))
        if kind == KIND_FP8B:    # random sign and magnitude codes below the NaN pattern; |w| ~ std with one common block scale
            mag = torch.randint(0, 0x78, (G, N, K), dtype=torch.uint8, device=device, generator=gen)
            sign = torch.randint(0, 2, (G, N, K), dtype=torch.uint8, device=device, generator=gen) << 7
            data = cut(mag | sign)
            sw = torch.full((hi - lo, -(-N // 128), -(-K // 128)), std / 60.0, dtype=torch.float32, device=device)
            return TcWeight(kind, hi - lo, N, K, data, encode_tmap(data, 128), sw)
        data = cut(torch.randint(0, 256, (G, N, K // 2), dtype=torch.uint8, device=device, generator=gen))
        vec = 16 if kind == KIND_NVFP4 else 32
        kstage = 128 if kind == KIND_W4A8 else 256
        nsf = (-(-N // 128) * 128) * (-(-K // kstage) * (kstage // vec))
        if kind == KIND_NVFP4:   # E4M3 scales in [0.5, 1.875]
            sf = cut(torch.randint(0x30, 0x40, (G, nsf), dtype=torch.uint8, device=device, generator=gen))
            alpha = torch.full((hi - lo,), std / 3.4 * act_gs, dtype=torch.float32, device=device)
        else:                    # UE8M0 scales 2^-7 .. 2^-6 -> |w| ~ std
            sf = cut(torch.randint(120, 122, (G, nsf), dtype=torch.uint8, device=device, generator=gen))
            alpha = torch.full((hi - lo,), std / 0.034, dtype=torch.float32, device=device)
        return TcWeight._finish(kind, hi - lo, N, K, data, sf, alpha, act_gs)

    @staticmethod
    def _finish(kind, G, N, K, data, sf, alpha, act_gs):
        sf_ptrs = torch.tensor([sf[g].data_ptr() for g in range(G)], dtype=torch.int64, device=data.device)
        inv = torch.tensor([1.0 / act_gs], dtype=torch.float32, device=data.device)
        return TcWeight(kind, G, N, K, data, encode_tmap(data, 128, unpack4=kind == KIND_W4A8), sf, sf_ptrs, alpha, inv)

    def dequantize(self) -> torch.Tensor:
        """fp32 [G, N, K] on CPU, without the activation scale folded into alpha (test helper)."""
        from ..ref import quant
        if self.kind in (KIND_BF16, KIND_F32):
            return self.data.float().cpu()
        if self.kind == KIND_FP8B:
            return torch.stack([quant.fp8_block_dequantize(self.data[g].cpu(), self.sf[g].cpu()) for g in range(self.G)])
        vec = 16 if self.kind == KIND_NVFP4 else 32
        kstage = 128 if self.kind == KIND_W4A8 else 256
        out = []
        for g in range(self.G):
            s = quant.unswizzle_sf_128x4(self.sf[g].cpu(), self.N, -(-self.K // kstage) * (kstage // vec))[:, :self.K // vec]
            if self.kind == KIND_NVFP4:
                gs = float(self.alpha[g]) * float(self.inv_act_gs[0])
                out.append(quant.nvfp4_dequantize(self.data[g].cpu(), s, gs))
            else:
                out.append(quant.mxfp4_dequantize(self.data[g].cpu(), s) * float(self.alpha[g]))
        return torch.stack(out)


@dataclass
class ActBuffer:
    """Activation operand for `tc_linear`: bf16 rows, or fp4 rows + row-major block scales, with its TMA
    descriptor for a token tile of `tn` rows."""
    kind: int
    rows: int
    K: int
    tn: int
    data: torch.Tensor
    tmap: torch.Tensor
    sf: torch.Tensor | None = None

    @staticmethod
    def alloc(kind: int, rows: int, K: int, tn: int, device) -> "ActBuffer":
        if kind == KIND_BF16:
            data = torch.zeros(rows, K, dtype=torch.bfloat16, device=device)
            return ActBuffer(kind, rows, K, tn, data, encode_tmap(data, tn))
        if kind == KIND_F32:
            return ActBuffer(kind, rows, K, tn, torch.zeros(rows, K, dtype=torch.float32, device=device), None)
        if kind == KIND_FP8B:    # E4M3 bytes + one fp32 scale per row and 128 channels
            data = torch.zeros(rows, K, dtype=torch.uint8, device=device)
            return ActBuffer(kind, rows, K, tn, data, encode_tmap(data, tn), torch.zeros(rows, -(-K // 128), dtype=torch.float32, device=device))
        if kind == KIND_W4A8:    # E4M3 bytes + one UE8M0 scale per row and 32 channels (scale rows padded to whole 128-channel stages)
            data = torch.zeros(rows, K, dtype=torch.uint8, device=device)
            return ActBuffer(kind, rows, K, tn, data, encode_tmap(data, tn), torch.zeros(rows, -(-K // 128) * 4, dtype=torch.uint8, device=device))
        vec = 16 if kind == KIND_NVFP4 else 32
        data = torch.zeros(rows, K // 2, dtype=torch.uint8, device=device)
        sf = torch.zeros(rows, -(-K // 256) * (256 // vec), dtype=torch.uint8, device=device)   # padded to whole stages
        return ActBuffer(kind, rows, K, tn, data, encode_tmap(data, tn), sf)

    @staticmethod
    def wrap_bf16(x: torch.Tensor, tn: int) -> "ActBuffer":
        _chk(x, torch.bfloat16, "x")
        return ActBuffer(KIND_BF16, x.shape[0], x.shape[1], tn, x, encode_tmap(x, tn))


SF_PER_STAGE = {KIND_NVFP4: 16, KIND_MXFP4: 8, KIND_W4A8: 4}        # weight block scales per row and pipeline stage


def pick_tn(rows: int, swiglu: bool = False) -> int:
    for tn in (16, 32, 64, 128):
        if rows <= tn:
            return tn
    return 128 if swiglu else 256


_SPLITK_WS: dict = {}
_SPLITK_KEEP: list = []        # outgrown scratch stays allocated: captured graphs still point at it


def _splitk_scratch(device, n_float: int, n_cnt: int):
    key = str(device)
    ws, cnt = _SPLITK_WS.get(key, (None, None))
    if ws is None or ws.numel() < n_float:
        _SPLITK_KEEP.append(ws)
        ws = torch.empty(max(n_float, 1 << 22), dtype=torch.float32, device=device)
    if cnt is None or cnt.numel() < n_cnt:
        _SPLITK_KEEP.append(cnt)
        cnt = torch.zeros(max(n_cnt, 1 << 16), dtype=torch.int32, device=device)
    _SPLITK_WS[key] = (ws, cnt)
    return ws, cnt


def tc_linear(w: TcWeight, x: ActBuffer, y: torch.Tensor | None, *, rows: int | None = None, w_up: TcWeight | None = None,
              residual: torch.Tensor | None = None, tiles: torch.Tensor | None = None, n_tiles: torch.Tensor | None = None,
              max_tiles: int = 0, splits: int = 1, status: torch.Tensor | None = None, max_ctas: int = 0,
              quant_out: ActBuffer | None = None, inv_gs_out: torch.Tensor | None = None, peer: dict | None = None, act: str | None = None,
              token_major: tuple | None = None, bound: float = 0.0, biases: tuple | None = None) -> torch.Tensor | None:
    """y[rows, N] = x[rows, K] @ w[g]^T (per tile's expert g when `tiles` is given).  `w_up` switches on the fused
    SwiGLU epilogue (y = silu(x w^T) * (x w_up^T)).  y is bf16 (optionally + residual) or fp32.  `quant_out` (an FP4
    activation buffer of the operands' kind, K = N) also receives the output quantised for the GEMM that follows
    (`inv_gs_out`: that GEMM's activation scale, NVFP4); y may then be None.
    `peer` fuses the hand-off to other GPUs into the epilogue: {"y": [device addresses of 1-2 peers' bf16 buffers], "ld": row
    pitch in elements, "row_map": int32 tensor or None (row r lands in row_map[r]), "flags": [peer flag addresses],
    "ctl": control block tensor, "done": zeroed uint32 counter tensor}; the flags are released with the step number
    once the whole output has been stored (y may be None when only the peers need the result).
    `act="relu2"`: squared ReLU on the output (an expert without a gate projection); `act="softcap"`: bound * tanh(y / bound);
    `act="clamped_glu"` (with `w_up`): gate and linear half with `biases` (fp32 [N] each), bounded by `bound`, g sigmoid(1.702 g) (u + 1)
    instead of SwiGLU.  `token_major=(rows per group, columns per group)`:
    a GEMM grouped over the heads of head-major operands (operand row = head * rows per group + token) writes head g's N columns of
    output row `token` at column g * columns per group."""
    rows = x.rows if rows is None else rows
    if w.kind != x.kind or w.K != x.K:
        raise ValueError("tc_linear: operand kinds / K differ")
    if y is None:
        epi = EPI_BF16
    else:
        epi = EPI_F32 if y.dtype == torch.float32 else (EPI_BF16_RESIDUAL if residual is not None else EPI_BF16)
    if w.kind == KIND_FP8B:
        if w_up is not None or tiles is not None or quant_out is not None or w.G != 1:
            raise ValueError("tc_linear: the FP8 block-scaled kernel is dense only (no SwiGLU / grouped / FP4 output)")
        if splits < 1 or (splits > 1 and x.tn > 64) or splits > (8 if x.tn == 16 else 4):
            splits = 1
        call("cuteafd_fp8_linear", x.tn, ptr(w.tmap), ptr(x.tmap), ptr(w.sf), ptr(x.sf), ptr(y), ptr(residual), y.stride(0), rows, w.N, w.K,
             epi, splits, ptr(status), stream())
        return y
    if w.kind == KIND_F32:
        if w_up is not None or residual is not None or quant_out is not None or peer is not None or y is None or y.dtype != torch.float32:
            raise ValueError("tc_linear: the fp32 kernel has a plain fp32 output only")
        gr, gc = token_major or (0, 0)
        call("cuteafd_f32_linear", ptr(x.data), x.data.stride(0), ptr(w.data), ptr(y), y.stride(0), ptr(tiles), ptr(n_tiles), max_tiles, rows, w.N, w.K,
             ACTIVATIONS[act], float(bound), gr, gc, ptr(w.alpha), stream())
        return y
    ws = cnt = None
    if splits > 1:
        n_items = -(-rows // x.tn)
        ws, cnt = _splitk_scratch(x.data.device, splits * rows * w.N, n_items * (-(-w.N // 128)) * 4)
    extra = None
    if quant_out is not None:
        if quant_out.kind != w.kind or quant_out.K != w.N:
            raise ValueError("tc_linear: quant_out must be an FP4 buffer of the operands' kind with K = N")
        extra = native.TcExtra()
        extra.q_out, extra.sf_out, extra.ldsf_out, extra.inv_gs_out = ptr(quant_out.data), ptr(quant_out.sf), quant_out.sf.shape[1], ptr(inv_gs_out)
    if act is not None or token_major is not None:
        extra = extra or native.TcExtra()
        extra.act, extra.act_p = ACTIVATIONS[act], float(bound)
        if biases is not None:
            _chk(biases[0], torch.float32, "biases"); _chk(biases[1], torch.float32, "biases")
            extra.bias, extra.bias2 = ptr(biases[0]), ptr(biases[1])
        extra.grp_rows, extra.grp_cols = token_major or (0, 0)
    if peer is not None:
        ys, fl = list(peer["y"]), list(peer["flags"])
        extra = extra or native.TcExtra()
        extra.n_peer, extra.peer_ld = len(ys), peer["ld"]
        for i in range(len(ys)):
            extra.peer_y[i], extra.peer_flag[i] = ys[i], fl[i]
        extra.peer_row_map, extra.peer_ctl, extra.peer_done = ptr(peer.get("row_map")), ptr(peer["ctl"]), ptr(peer["done"])
    call("cuteafd_tc_linear", w.kind, 1 if w_up is not None else 0, x.tn, ptr(w.tmap), ptr(w_up.tmap) if w_up else None,
         ptr(x.tmap), ptr(w.sf_ptrs), ptr(w_up.sf_ptrs) if w_up else None, ptr(x.sf), x.sf.shape[1] if x.sf is not None else 0,
         ptr(w.alpha), ptr(w_up.alpha) if w_up else None, ptr(tiles), ptr(n_tiles), max_tiles, ptr(y), ptr(residual),
         y.stride(0) if y is not None else 0, rows, w.N, w.K, epi, splits, ptr(ws), ptr(cnt), ptr(status), max_ctas,
         ctypes.byref(extra) if extra is not None else None, stream())
    return y


# ------------------------------------------------------------------ EXL3 (trellis) weights
@dataclass
class Exl3Weight:
    """One EXL3 linear as shipped: trellis uint16 [K/16, N/16, 16*bits], suh fp16 [K], svh fp16 [N] (y = x @ W)."""
    trellis: torch.Tensor
    suh: torch.Tensor
    svh: torch.Tensor

    @property
    def K(self) -> int:
        return self.trellis.shape[0] * 16

    @property
    def N(self) -> int:
        return self.trellis.shape[1] * 16

    @property
    def bits(self) -> int:
        return self.trellis.shape[2] // 16


_EXL3_WS: dict = {}


def exl3_linear(w: Exl3Weight, x: torch.Tensor, y: torch.Tensor, *, rows: int | None = None, residual: torch.Tensor | None = None,
                k_splits: int = 0) -> torch.Tensor:
    """y[rows, N] = x[rows, K] @ W(+ residual) with W decoded from the trellis inside the GEMM (decode-sized batches)."""
    _chk(x, torch.bfloat16, "x")
    rows = x.shape[0] if rows is None else rows
    K, N = w.K, w.N
    if not k_splits:      # enough warps to fill the machine: N/16 strips x splits ~ 4 per SM sub-partition
        k_splits = max(1, min(K // 256, -(-148 * 16 // (N // 16))))
    pad = -(-rows // 16) * 16
    key = str(x.device)
    xr, part = _EXL3_WS.get(key, (None, None))
    if xr is None or xr.numel() < pad * K:
        xr = torch.empty(max(pad * K, 1 << 20), dtype=torch.float16, device=x.device)
    if part is None or part.numel() < k_splits * pad * N:
        part = torch.empty(max(k_splits * pad * N, 1 << 22), dtype=torch.float32, device=x.device)
    _EXL3_WS[key] = (xr, part)
    call("cuteafd_exl3_linear", ptr(x), ptr(w.trellis), ptr(w.suh), ptr(w.svh), ptr(residual), ptr(y), ptr(xr), ptr(part), rows, K, N, w.bits,
         k_splits, y.stride(0), stream())
    return y


# ------------------------------------------------------------------ elementwise
def embed_gather(tokens: torch.Tensor, table: torch.Tensor, out: torch.Tensor, status: torch.Tensor | None = None):
    _chk(tokens, torch.int32, "tokens"); _chk(table, torch.bfloat16, "table")
    call("cuteafd_embed_gather", ptr(tokens), ptr(table), ptr(out), tokens.numel(), table.shape[1], table.shape[0], ptr(status), stream())
    return out


def add_rmsnorm(x: torch.Tensor, delta: torch.Tensor | None, w: torch.Tensor, y: torch.Tensor | None, eps: float, rows: int | None = None,
                quant: "ActBuffer | None" = None, inv_gs: torch.Tensor | None = None):
    """x += delta (if given, in place); y = rmsnorm(x) * w.  With `quant` (an FP4 activation buffer) the normalised
    rows are also written quantised in the same launch (y may then be None)."""
    _chk(x, torch.bfloat16, "x"); _chk(w, torch.float32, "w")
    n = x.shape[0] if rows is None else rows
    if quant is not None and quant.kind in FUSED_QUANT_KINDS:
        call("cuteafd_add_rmsnorm_quant", ptr(x), ptr(delta), ptr(w), ptr(y), n, x.shape[1], eps, ptr(quant.data), ptr(quant.sf),
             quant.sf.shape[1], ptr(inv_gs), _QKIND[quant.kind], stream())
    else:
        call("cuteafd_add_rmsnorm", ptr(x), ptr(delta), ptr(w), ptr(y), n, x.shape[1], eps, stream())
    return y


def qk_norm_rope_kvwrite(qkv, positions, slot_map, q_norm, k_norm, kv_cache, T, Hq, Hkv, D, theta, interleaved, eps, status=None):
    n_slots = kv_cache.shape[0]
    call("cuteafd_qk_norm_rope_kvwrite", ptr(qkv), ptr(positions), ptr(slot_map), ptr(q_norm), ptr(k_norm), ptr(kv_cache),
         T, Hq, Hkv, D, theta, 1 if interleaved else 0, eps, n_slots, ptr(status), stream())


def quant_fp4_rows(x: torch.Tensor, out: ActBuffer, *, src_rows: torch.Tensor | None = None, n_rows_dev: torch.Tensor | None = None,
                   rows: int | None = None, inv_gs: torch.Tensor | None = None):
    _chk(x, torch.bfloat16, "x")
    if out.kind == KIND_W4A8:
        call("cuteafd_act_quant_fp8_ue8m0", ptr(x), ptr(src_rows), ptr(n_rows_dev), ptr(out.data), ptr(out.sf), out.rows if rows is None else rows,
             out.K, x.stride(0), out.sf.shape[1], stream())
        return out
    if out.kind == KIND_FP8B:
        if src_rows is not None or n_rows_dev is not None:
            raise ValueError("FP8 activation quantisation has no gather form")
        call("cuteafd_act_quant_fp8_block128", ptr(x), ptr(out.data), ptr(out.sf), out.rows if rows is None else rows, out.K, x.stride(0), stream())
        return out
    call("cuteafd_quant_fp4_rows", 1 if out.kind == KIND_MXFP4 else 0, ptr(x), ptr(src_rows), ptr(n_rows_dev), ptr(out.data),
         ptr(out.sf), out.rows if rows is None else rows, out.K, x.stride(0), out.sf.shape[1], ptr(inv_gs), stream())
    return out


def gather_rows(x, src_rows, n_rows_dev, out, rows):
    call("cuteafd_gather_rows", ptr(x), ptr(src_rows), ptr(n_rows_dev), ptr(out), rows, x.shape[1], stream())
    return out


def kv_pages_copy(kv, pairs, pool, to_pool: bool):
    """Moves KV pages between the device store `kv` [layers, slots, ...] and a slab pool [slabs, layers, page...] (device
    memory or pinned host memory) in one launch.  `pairs` is an int32 device tensor [n, 2] of (device page, slab)."""
    L = kv.shape[0]
    page_bytes = pool[0, 0].numel() * pool.element_size()
    assert pool.shape[1] == L and kv.is_contiguous() and pool.is_contiguous() and pairs.dtype == torch.int32 and pairs.is_cuda
    call("cuteafd_kv_pages_copy", ptr(kv), kv.stride(0) * kv.element_size(), L, page_bytes, ptr(pairs), pairs.shape[0], pool.data_ptr(),
         pool.stride(0) * pool.element_size(), 0 if to_pool else 1, stream())


def l2_prefetch(t):
    """Hints the memory system to pull a tensor (e.g. the next layer's weights) into L2; returns immediately."""
    call("cuteafd_l2_prefetch", ptr(t), t.numel() * t.element_size(), stream())


def act_quant_fp8_ue8m0(x, q, sf):
    call("cuteafd_act_quant_fp8_ue8m0", ptr(x), None, None, ptr(q), ptr(sf), x.shape[0], x.shape[1], x.stride(0), sf.shape[1], stream())


def silu_mul(g, u, out, limit: float = 0.0):
    call("cuteafd_silu_mul", ptr(g), ptr(u), ptr(out), g.numel(), limit, stream())
    return out


def router_logits(x, w: "TcWeight", logits, T: int):
    """fp32 router logits of `T` token rows (bf16 `x` [rows, H]) against a bf16 router weight [E, H]: the SIMT kernel for
    decode-sized batches (the tensor-core GEMM is launch- and cluster-overhead bound at this size)."""
    assert w.kind == KIND_BF16 and w.G == 1 and x.dtype == torch.bfloat16 and x.stride(0) == w.K and logits.stride(0) == w.N
    call("cuteafd_router_logits", ptr(x), ptr(w.data), ptr(logits), T, w.N, w.K, stream())
    return logits


# ------------------------------------------------------------------ MoE control
def scoring_code(scoring: str, group_score: str = "top2") -> int:
    return SCORING[scoring] | (GROUP_BY_MAX if group_score == "max" else 0)


def router_select(logits, bias, idx, wts, T, k, scoring, normalize, route_scale, n_group=1, topk_group=1, group_score="top2"):
    _chk(logits, torch.float32, "logits")
    call("cuteafd_router_select", ptr(logits), ptr(bias), ptr(idx), ptr(wts), T, logits.shape[1], k, scoring_code(scoring, group_score),
         1 if normalize else 0, route_scale, n_group, topk_group, stream())


_TICKETS: dict = {}


def router_select_pack(logits, bias, idx, wts, T, k, scoring, normalize, route_scale, n_group, topk_group,
                       src_token, slot_row, counts, offsets, tiles, n_tiles, n_rows, e_lo, e_hi, tn, max_tiles, src_route=None, group_score="top2"):
    """`router_select` followed by `route_pack` in one launch (the select block that finishes last packs)."""
    _chk(logits, torch.float32, "logits")
    dev = logits.device
    if dev not in _TICKETS:
        _TICKETS[dev] = torch.zeros(1, dtype=torch.int32, device=dev)
    call("cuteafd_router_select_pack", ptr(logits), ptr(bias), ptr(idx), ptr(wts), T, logits.shape[1], k, scoring_code(scoring, group_score),
         1 if normalize else 0, route_scale, n_group, topk_group, ptr(src_token), ptr(slot_row), ptr(counts), ptr(offsets),
         ptr(tiles), ptr(n_tiles), ptr(n_rows), e_lo, e_hi, tn, max_tiles, ptr(src_route), ptr(_TICKETS[dev]), stream())


def router_fused(x, w: "TcWeight", logits, bias, idx, wts, T, k, scoring, normalize, route_scale, n_group=1, topk_group=1, pack: dict | None = None):
    """The whole router of a decode-sized step in one launch: fp32 logits of `T` bf16 rows against the bf16 router weight, top-k
    selection with gate weights, and - with `pack` (src_token, slot_row, counts, offsets, tiles, n_tiles, n_rows, e_lo, e_hi, tn,
    max_tiles, optional src_route) - the expert-order route packing and tile table."""
    assert w.kind == KIND_BF16 and w.G == 1 and x.dtype == torch.bfloat16 and x.stride(0) == w.K and logits.stride(0) == w.N
    dev = logits.device
    if dev not in _TICKETS:
        _TICKETS[dev] = torch.zeros(1, dtype=torch.int32, device=dev)
    pk = pack or {}
    g = lambda name: ptr(pk.get(name))
    call("cuteafd_router_fused", ptr(x), ptr(w.data), ptr(logits), ptr(bias), ptr(idx), ptr(wts), T, w.N, w.K, k, SCORING[scoring],
         1 if normalize else 0, route_scale, n_group, topk_group, g("src_token"), g("slot_row"), g("counts"), g("offsets"), g("tiles"),
         g("n_tiles"), g("n_rows"), pk.get("e_lo", 0), pk.get("e_hi", 0), pk.get("tn", 1), pk.get("max_tiles", 0), g("src_route"),
         ptr(_TICKETS[dev]), stream())


def route_pack(idx, src_token, slot_row, counts, offsets, tiles, n_tiles, n_rows, T, k, e_lo, e_hi, tn, max_tiles, src_route=None, *,
               wait=None, lane_T=None, t_cap: int = 0):
    """Packs the routes of `T` tokens into expert order.  `wait` (a `native.FlagWaitArg`) makes the kernel wait for the peers
    that deliver the routing table; `lane_T` (int32 device tensor, one count per lane) + `t_cap` describe a table of several
    senders laid out [lane][t_cap][k] (T = lanes * t_cap) whose rows beyond each lane's count are skipped."""
    call("cuteafd_route_pack", ptr(idx), ptr(src_token), ptr(slot_row), ptr(counts), ptr(offsets), ptr(tiles), ptr(n_tiles),
         ptr(n_rows), T, k, e_lo, e_hi, tn, max_tiles, ptr(src_route), ctypes.byref(wait) if wait is not None else None,
         ptr(lane_T), t_cap, stream())


def route_gather(src_q, src_sf, src_token, n_rows, dst: "ActBuffer", rows_cap: int, status=None):
    """dst row c = slab row src_token[c] (payload and block scales) for c < n_rows: token-major slab -> expert order."""
    row_bytes = src_q.shape[-1] * src_q.element_size()
    sf_bytes = src_sf.shape[-1] if src_sf is not None else 0
    call("cuteafd_route_gather", ptr(src_q), ptr(src_sf), ptr(src_token), ptr(n_rows), ptr(dst.data), ptr(dst.sf) if src_sf is not None else None,
         row_bytes, sf_bytes, sf_bytes, dst.sf.shape[1] if src_sf is not None else 0, src_q.numel() * src_q.element_size() // row_bytes,
         rows_cap, ptr(status), stream())
    return dst


def router_hash_select(logits, tid2eid, tokens, idx, wts, T, k, route_scale: float = 1.0, status=None):
    """Hash routing: experts of token row t are tid2eid[tokens[t]] ([vocab, k] int32); gate weights are the normalised
    sqrt-softplus scores of `logits` at those experts times `route_scale`."""
    _chk(logits, torch.float32, "logits"); _chk(tid2eid, torch.int32, "tid2eid"); _chk(tokens, torch.int32, "tokens")
    call("cuteafd_router_hash_select", ptr(logits), ptr(tid2eid), ptr(tokens), ptr(idx), ptr(wts), T, logits.shape[1], k, tid2eid.shape[0],
         route_scale, ptr(status), stream())


def moe_combine(y, slot_row, wts, shared, residual, out, T, k, *, norm_w=None, eps: float = 0.0, xn=None, quant=None, inv_gs=None, wait=None):
    """out = residual + shared + sum_slot w * y[slot_row].  With `norm_w` the same launch also applies the next
    layer's RMSNorm to `out`, written as bf16 (`xn`) and/or FP4 (`quant`, an activation buffer).  `wait` (a
    `native.FlagWaitArg`): the kernel first waits for the peers that deliver `y`."""
    w = ctypes.byref(wait) if wait is not None else None
    if norm_w is None:
        call("cuteafd_moe_combine", ptr(y), ptr(slot_row), ptr(wts), ptr(shared), ptr(residual), ptr(out), T, y.shape[1], k, w, stream())
        return out
    fp4 = quant is not None and quant.kind in FUSED_QUANT_KINDS
    call("cuteafd_moe_combine_norm", ptr(y), ptr(slot_row), ptr(wts), ptr(shared), ptr(residual), ptr(out), T, y.shape[1], k, ptr(norm_w),
         eps, ptr(xn), ptr(quant.data) if fp4 else None, ptr(quant.sf) if fp4 else None, quant.sf.shape[1] if fp4 else 0,
         ptr(inv_gs) if fp4 else None, _QKIND[quant.kind] if fp4 else 0, w, stream())
    return out


# ------------------------------------------------------------------ attention
def paged_attention(q, kv, page_table, kv_len, q_start, q_len, out, *, T, n_seq, max_q_len, q_stride, Hq, Hkv, D, n_splits=1,
                    part_o=None, part_ml=None, window=0, sink=None, scale=None):
    call("cuteafd_paged_attention", ptr(q), ptr(kv), ptr(page_table), ptr(kv_len), ptr(q_start), ptr(q_len), ptr(sink), ptr(out),
         ptr(part_o), ptr(part_ml), T, n_seq, max_q_len, q_stride, Hq, Hkv, D, page_table.shape[1], n_splits, window,
         float(scale if scale is not None else D ** -0.5), stream())
    return out


def encode_kv_tmaps(kv: torch.Tensor) -> torch.Tensor:
    """TMA descriptors (uint8 [layers, 128]) for a paged K/V store [layers, slots, 2, Hkv, 128] bf16."""
    _chk(kv, torch.bfloat16, "kv")
    L, slots, two, Hkv, D = kv.shape
    if D != 128 or two != 2:
        raise ValueError("tensor-core attention needs head_dim 128")
    host = torch.zeros(L, 128, dtype=torch.uint8)
    for l in range(L):
        call("cuteafd_tmap_encode_kv", host[l].data_ptr(), kv[l].data_ptr(), Hkv, slots)
    return host.to(kv.device)


def paged_attention_tc(q, kv_map, page_table, kv_len, q_start, q_len, out, *, T, n_seq, max_q_len, q_stride, Hq, Hkv,
                       n_splits=1, part_o=None, part_ml=None, window=0, sink=None, scale=None, status=None, quant=None, inv_gs=None,
                       partials_only=False) -> bool:
    """Tensor-core (tcgen05) paged attention for head_dim 128; `kv_map` is one row of `encode_kv_tmaps`.
    `quant` (an FP4 activation buffer): with split-KV the merge also writes the output rows quantised for the output
    projection.  Returns True when that happened (False: the caller quantises `out` itself).
    `partials_only` (context split, needs n_splits >= 2): leave the unnormalised split outputs in `part_o` / `part_ml`
    ([n_splits, T, Hq, 128] / [n_splits, T, Hq, 2]) and do not merge; `attn_merge` finishes over all owners' partials."""
    fused = quant is not None and quant.kind in FP4_KINDS and n_splits > 1 and (Hq * 128) % 256 == 0 and not partials_only
    if partials_only:
        call("cuteafd_attn_partials_only")
    call("cuteafd_paged_attention_tc", ptr(q), ptr(kv_map), ptr(page_table), ptr(kv_len), ptr(q_start), ptr(q_len), ptr(sink),
         ptr(out), ptr(part_o), ptr(part_ml), T, n_seq, max_q_len, q_stride, Hq, Hkv, page_table.shape[1], n_splits, window,
         float(scale if scale is not None else 128 ** -0.5), ptr(status), ptr(quant.data) if fused else None,
         ptr(quant.sf) if fused else None, quant.sf.shape[1] if fused else 0, ptr(inv_gs) if fused else None,
         (2 if quant.kind == KIND_MXFP4 else 1) if fused else 0, stream())
    return fused


def attn_merge(part_o, part_ml, out, *, T, Hq, n_parts, sink=None):
    """Merges `n_parts` attention partials laid side by side (unnormalised outputs [n_parts, T, Hq, 128] fp32 and
    (max, sum) pairs [n_parts, T, Hq, 2]) into `out` [T, Hq * 128] bf16.  With a context split the parts are the
    splits of every GPU that owns a piece of the context."""
    call("cuteafd_attn_merge", ptr(part_o), ptr(part_ml), ptr(sink), ptr(out), T, Hq, n_parts, stream())
    return out


def context_split_attention(q, kv_maps, page_tables, kv_lens, q_start, q_len, out, *, T, n_seq, Hq, Hkv, splits_per_part=2, scale=None,
                            status=None, sink=None):
    """Decode attention over a context whose pages are held in several paged stores (one per owner): partial attention
    per owner, then one merge.  On one GPU the owners are just different stores, which is how the path is tested; across
    GPUs every owner runs its own part and ships its `part_o` / `part_ml` slices to the merging rank with the peer copy.
    Decode rows only (one query token per sequence): every cached key is visible, so each owner passes its own length."""
    n_own = len(kv_maps)
    s = splits_per_part
    part_o = torch.empty(n_own * s * T * Hq * 128, dtype=torch.float32, device=q.device)
    part_ml = torch.empty(n_own * s * T * Hq * 2, dtype=torch.float32, device=q.device)
    for o in range(n_own):
        po = part_o[o * s * T * Hq * 128:(o + 1) * s * T * Hq * 128]
        pm = part_ml[o * s * T * Hq * 2:(o + 1) * s * T * Hq * 2]
        paged_attention_tc(q, kv_maps[o], page_tables[o], kv_lens[o], q_start, q_len, out, T=T, n_seq=n_seq, max_q_len=1, q_stride=q.stride(0),
                           Hq=Hq, Hkv=Hkv, n_splits=s, part_o=po, part_ml=pm, scale=scale, status=status, partials_only=True)
    return attn_merge(part_o, part_ml, out, T=T, Hq=Hq, n_parts=n_own * s, sink=sink)


# ------------------------------------------------------------------ sampling
def argmax_rows(logits, tok, *, rows=None, V=None, masks=None, logprob=None, status=None):
    _chk(logits, torch.float32, "logits")
    call("cuteafd_argmax_rows", ptr(logits), logits.stride(0), logits.shape[0] if rows is None else rows,
         logits.shape[1] if V is None else V, ptr(masks), masks.shape[1] if masks is not None else 0, ptr(tok), ptr(logprob),
         ptr(status), stream())
    return tok


def pack_sample_params(params_list, positions) -> torch.Tensor:
    """[(temperature, top_p, top_k, min_p, seed)], positions -> uint8 [T, 32] host tensor for `sample_rows`."""
    import struct
    buf = bytearray()
    for p, pos in zip(params_list, positions):
        buf += struct.pack("<fffiQQ", p.temperature, p.top_p, p.min_p, p.top_k, p.seed & (2 ** 64 - 1), int(pos))
    return torch.frombuffer(buf, dtype=torch.uint8).reshape(-1, 32).clone()


def sample_rows(logits, params_dev, tok, status, *, masks=None):
    _chk(logits, torch.float32, "logits")
    call("cuteafd_sample_rows", ptr(logits), logits.stride(0), logits.shape[0], logits.shape[1], ptr(masks),
         masks.shape[1] if masks is not None else 0, ptr(params_dev), ptr(tok), ptr(status), stream())
    return tok


def verify_accept(inputs, target, n_drafts, accepted, n_emit, eos: int = -1):
    n_seq, width = inputs.shape
    call("cuteafd_verify_accept", ptr(inputs), ptr(target), ptr(n_drafts), ptr(accepted), ptr(n_emit), n_seq, width, eos, stream())


# ------------------------------------------------------------------ linear attention (GDN / KDA recurrent layers)
def gated_delta_step(q, k, v, g, beta, state, slot_of_seq, q_start, q_len, out, *, snapshots=None, status=None):
    """Gated delta rule over runs of tokens: q, k, v, out bf16 [T, H, 128]; g fp32 [T, H] (decay per head) or [T, H, 128] (per key
    channel); beta fp32 [T, H]; state fp32 [slots, H, 128, 128] updated in place for the slots named by `slot_of_seq`; run s covers
    rows [q_start[s], q_start[s] + q_len[s]).  `snapshots` (fp32 [T, H, 128, 128]) receives the state after every token."""
    _chk(q, torch.bfloat16, "q"); _chk(k, torch.bfloat16, "k"); _chk(v, torch.bfloat16, "v"); _chk(out, torch.bfloat16, "out")
    _chk(g, torch.float32, "g"); _chk(beta, torch.float32, "beta"); _chk(state, torch.float32, "state")
    T, H, D = q.shape
    if D != 128 or v.shape[-1] != 128 or state.shape[1:] != (H, 128, 128):
        raise ValueError("gated_delta_step: heads are 128 x 128")
    call("cuteafd_gated_delta_step", ptr(q), ptr(k), ptr(v), ptr(g), ptr(beta), ptr(state), ptr(slot_of_seq), ptr(q_start), ptr(q_len), ptr(out),
         ptr(snapshots), slot_of_seq.numel(), H, 1 if g.dim() == 3 else 0, state.shape[0], ptr(status), stream())
    return out


def short_conv4(x, w, carry, slot_of_seq, q_start, q_len, y, *, status=None):
    """Causal depthwise convolution of width 4 + SiLU: x, y bf16 [T, C]; w fp32 [C, 4]; carry bf16 [slots, 3, C] (the last three
    inputs of every sequence, updated in place)."""
    _chk(y, torch.bfloat16, "y"); _chk(w, torch.float32, "w"); _chk(carry, torch.bfloat16, "carry")      # x may be a column slice of wider rows
    call("cuteafd_short_conv4", ptr(x), ptr(w), ptr(carry), ptr(slot_of_seq), ptr(q_start), ptr(q_len), ptr(y), slot_of_seq.numel(), y.shape[1],
         x.stride(0), carry.shape[0], ptr(status), stream())
    return y


def compress_pool(kv, scores, state, state_slot, q_start, q_len, pos0, out_start, norm_w, out, *, n_seq: int, max_blocks: int, ratio: int,
                  eps: float = 1e-6):
    """Softmax pooling of KV candidate rows into one compressed cache row per `ratio` positions (see csrc/compressor.cu): fp32
    kv / scores [T, D], per-sequence open-block state [slots, 3, D], int32 step descriptors per sequence; rows of the blocks completed
    in this step land in `out` (bf16 [n, D]) from `out_start[s]` on.  `max_blocks`: the most blocks any sequence touches in the step."""
    call("cuteafd_compress_pool", ptr(kv), ptr(scores), ptr(state), ptr(state_slot), ptr(q_start), ptr(q_len), ptr(pos0), ptr(out_start),
         ptr(norm_w), ptr(out), n_seq, max_blocks, kv.shape[1], ratio, eps, stream())
    return out


# ------------------------------------------------------------------ layer stacks: row kernels between two matrix products
def emit_arg(norm=None, xn=None, cat=None):
    """What the row kernels below leave for the next product.  `norm` = (w, b, alpha) of a Dynamic Tanh, written to `xn`; `cat`: buffer
    whose leading columns take the plain row."""
    e = native.EmitArg()
    if norm is not None:
        e.w, e.b, e.alpha, e.xn, e.ldn = ptr(norm[0]), ptr(norm[1]), float(norm[2]), ptr(xn), xn.stride(0)
    if cat is not None:
        e.cat, e.ldc = ptr(cat), cat.stride(0)
    return e


def _f32(t) -> int:
    return 1 if t.dtype == torch.float32 else 0


def stack_embed(tokens, positions, table, pos_table, x, x0, emit, T: int, *, f32: bool, status=None):
    """x[t] = table[token] + pos_table[position] (fp32 rows); `x0`: view whose rows take the same values as matrix operand."""
    _chk(tokens, torch.int32, "tokens"); _chk(table, torch.bfloat16, "table"); _chk(x, torch.float32, "x")
    call("cuteafd_stack_embed", ptr(tokens), ptr(positions), ptr(table), ptr(pos_table), ptr(x), ptr(x0), x0.stride(0) if x0 is not None else 0, T,
         x.shape[1], table.shape[0], pos_table.shape[0] if pos_table is not None else 0, 1 if f32 else 0, ctypes.byref(emit), ptr(status), stream())


def stack_stream(x, emit, T: int, *, f32: bool, vec=None, src_rows=None):
    """Rows x[t] (+ `vec`, written back), or the rows listed in `src_rows`, handed on by `emit`."""
    _chk(x, torch.float32, "x")
    call("cuteafd_stack_stream", ptr(x), ptr(vec), ptr(src_rows), T, x.shape[1], 1 if f32 else 0, ctypes.byref(emit), stream())


def stack_combine(x, mix, ls1, y, slot_row, wts, ls2, emit, T: int, k: int):
    """x += ls1 * mix + ls2 * sum over the token's k routes of wts * y[slot_row]; the new rows are handed on by `emit`."""
    _chk(x, torch.float32, "x")
    call("cuteafd_stack_combine", ptr(x), ptr(mix), ptr(ls1), ptr(y), ptr(slot_row), ptr(wts), ptr(ls2), T, x.shape[1], k, _f32(mix),
         ctypes.byref(emit) if emit is not None else None, stream())


def latent_prepare(proj, norm_w, slot_map, q, cache, gate, logits, tiles, n_tiles, *, T, ldt, H, d, r, rp, E, tn, eps, status=None):
    """Splits the fused projection rows (queries | latent | gates | router logits, fp32): queries head-major [H, ldt, q.shape[-1]], the
    RMS-normed latent into the paged cache, sigmoid gates, compact router logits, and the tile table of the per-head products."""
    _chk(proj, torch.float32, "proj")
    call("cuteafd_latent_prepare", ptr(proj), proj.stride(0), ptr(norm_w), ptr(slot_map), ptr(q), ptr(cache), ptr(gate), ptr(logits), ptr(tiles),
         ptr(n_tiles), T, ldt, H, d, q.shape[-1], r, rp, cache.stride(0), cache.shape[0], E, tn, eps, _f32(q), ptr(status), stream())


def latent_attention(q_lat, kv_map, page_table, kv_len, q_start, q_len, gate, out, *, T, ldt, n_seq, max_q_len, H, rank_pad, n_splits=1, part_o=None,
                     part_ml=None, scale, q_rope=None, sink=None, status=None):
    """Absorbed latent attention over the paged cache (tcgen05); q_lat, out: head-major [H, ldt, rank_pad] bf16.  `q_rope` [H, ldt, 64]: rotated parts
    (the rows' 64 columns behind the latent are the rotated key); `sink` fp32 [H]: one more logit per head."""
    call("cuteafd_latent_attention", ptr(q_lat), ptr(q_rope), ptr(sink), ptr(kv_map), ptr(page_table), ptr(kv_len), ptr(q_start), ptr(q_len), ptr(gate), ptr(out), ptr(part_o),
         ptr(part_ml), T, ldt, n_seq, max_q_len, H, rank_pad, page_table.shape[1], n_splits, float(scale), ptr(status), stream())


def latent_attention_simt(q_lat, cache, page_table, kv_len, q_start, q_len, gate, out, *, T, ldt, n_seq, H, rank_pad, scale, q_rope=None, sink=None, status=None):
    """The same on the ordinary cores: fp32 operands, latents wider than 512, more than 128 heads, rotated parts [H, ldt, any multiple of 8]."""
    call("cuteafd_latent_attention_simt", ptr(q_lat), ptr(q_rope), q_rope.shape[-1] if q_rope is not None else 0, ptr(sink), ptr(cache), ptr(page_table), ptr(kv_len), ptr(q_start), ptr(q_len), ptr(gate), ptr(out), T, ldt,
         n_seq, H, rank_pad, cache.stride(0), page_table.shape[1], cache.shape[0], float(scale), _f32(q_lat), ptr(status), stream())


def latent_down(proj, q_col: int, kv_col: int, q_norm, kv_norm, rope, slot_map, cq, cache, *, T, r, rp, rot, eps, status=None):
    """Splits fused down-projection rows (fp32: the queries' latent from column `q_col`, the latent and the rotated key part from `kv_col`): the RMS-normed
    queries' latent into `cq` [., q_rank_pad], the normed latent and the rotated part (neighbouring pairs) into the paged cache rows."""
    _chk(proj, torch.float32, "proj")
    a = native.LatentDown()
    a.proj, a.q_norm, a.kv_norm, a.rope, a.slot_map, a.cq, a.cache, a.status = (ptr(t) for t in (proj, q_norm, kv_norm, rope, slot_map, cq, cache, status))
    a.ldp, a.q_col, a.kv_col, a.q_rank, a.ldq, a.r, a.rp, a.rot, a.rotp = proj.stride(0), q_col, kv_col, q_norm.numel(), cq.stride(0), r, rp, rot, -(-rot // 64) * 64
    a.row_stride, a.n_slots, a.T, a.eps = cache.stride(0), cache.shape[0], T, eps
    call("cuteafd_latent_down", ctypes.addressof(a), _f32(cq), stream())


def latent_split(q, rope, qn, qr, tiles, n_tiles, *, T, ldt, H, d, rot, tn):
    """Expanded query rows [T, H * (d + rot)] -> head-major unrotated parts [H, ldt, qn.shape[-1]], rotated parts [H, ldt, qr.shape[-1]] (neighbouring
    pairs) and the tile table of the products grouped over heads."""
    call("cuteafd_latent_split", ptr(q), q.stride(0), ptr(rope), ptr(qn), ptr(qr), ptr(tiles), ptr(n_tiles), T, ldt, H, d, qn.shape[-1], rot, qr.shape[-1] if qr is not None else 0, tn,
         _f32(q), stream())


# ------------------------------------------------------------------ hybrid stacks: norms around sub-layers, short convolutions, recurrence, windows
ROWS_EMBED, ROWS_ADD, ROWS_GATHER = 0, 1, 2


def norm_rows(x, W: int, rows: int, *, f32: bool, eps: float, gain=None, xn=None, tokens=None, table=None, add=None, bias=None, post=None, mult: float = 1.0,
              src_rows=None, scale: float = 1.0, raw: bool = False, status=None):
    """Residual rows (fp32 [., Wp], norms average over W): x += mult * norm(add + bias) with `add` (`post`: gain of that norm, None = no norm), and with
    `tokens` and `table` besides + scale * table[token]; x = scale * table[token] with `tokens` alone; the rows listed in `src_rows` otherwise.  `xn`
    receives the rows RMS-normed with `gain` (None: without gains), or as they are (`raw`)."""
    _chk(x, torch.float32, "x")
    a = native.NormRows()
    a.x, a.W, a.Wp, a.eps, a.mult, a.status = ptr(x), W, x.shape[1], eps, mult, ptr(status)
    a.gain, a.xn, a.ldn, a.scale, a.raw = ptr(gain), ptr(xn), xn.stride(0) if xn is not None else 0, float(scale), 1 if raw else 0
    mode = ROWS_GATHER
    if tokens is not None:
        _chk(tokens, torch.int32, "tokens"); _chk(table, torch.bfloat16, "table")
        if table.shape[1] != x.shape[1]:
            raise ValueError("norm_rows: table and residual rows differ in width")
        mode, a.tokens, a.table, a.vocab = ROWS_EMBED, ptr(tokens), ptr(table), table.shape[0]
    if add is not None:
        if add.shape[1] != x.shape[1]:
            raise ValueError("norm_rows: added rows and residual rows differ in width")
        mode, a.add, a.bias, a.post = ROWS_ADD, ptr(add), ptr(bias), ptr(post)
    elif tokens is None:
        a.src_rows = ptr(src_rows)
    call("cuteafd_norm_rows", ctypes.addressof(a), mode, rows, 1 if f32 else 0, stream())


def rope_table(positions, freq, amp: float, out, T: int):
    """Cosine / sine rows [T, pairs] of the step's positions; `freq` fp32 [2, pairs] (value, rounding error)."""
    _chk(positions, torch.int32, "positions"); _chk(freq, torch.float32, "freq")
    call("cuteafd_rope_table", ptr(positions), ptr(freq), float(amp), freq.shape[1], ptr(out), T, stream())


QK_NORMS = {"": 0, "head": 1, "whole": 2}


def conv_qkv(proj, w, q_norm, k_norm, rope, ring, q, cache, meta: dict, *, H, G, dim, dp, vdim, dvp, pairs, eps, n_seq, max_q_len, bias=None, norm: str = "head",
             half: bool = False, values_are_keys: bool = False, n_slots: int = 0, pooled=None, pool: int = 0, status=None):
    """Short causal convolution over projected query / key / value rows (+ `bias`), norms, rotation; queries to `q` [., H * dp], keys and values to
    the paged `cache` rows.  `w` None: no convolution.  `ring` [slots, depth + taps - 1, channels]: inputs by position (None with one tap: give the
    number of state slots).  `norm`: "head" (gains [dim], None: without), "whole" (over all heads at once, gains [H * dim] / [G * dim]) or "".  `half`: dimensions i
    and i + pairs turn together instead of neighbours.  `values_are_keys`: no value channels, the keys in front of norm and rotation are the values.
    `pooled`, `pool`: rows of the pooled blocks of that many tokens (see `pool_kv`), of which short runs leave those that they complete.
    `meta`: the step's device inputs.  G = 0: queries only."""
    if w is not None:
        _chk(w, torch.float32, "w")
    a = native.ConvQkv()
    a.proj, a.w, a.bias, a.q_norm, a.k_norm, a.rope, a.ring, a.q, a.cache, a.status = (ptr(t) for t in (proj, w, bias, q_norm, k_norm, rope, ring, q, cache, status))
    a.norm, a.half, a.v_from_k = QK_NORMS[norm], 1 if half else 0, 1 if values_are_keys else 0
    for n in ("state_slot", "q_start", "q_len", "kv_len", "slot_map"):
        setattr(a, n, ptr(meta[n]))
    a.ldp, a.q_stride, a.H, a.G, a.dim, a.dp, a.vdim, a.dvp, a.pairs, a.eps = proj.stride(0), q.stride(0), H, G, dim, dp, vdim, dvp, pairs, eps
    a.row_stride, a.n_slots = (cache.stride(0), cache.shape[0]) if cache is not None else (8, 0)
    a.taps, a.C, a.n_seq, a.max_q_len = w.shape[0] if w is not None else 1, (H + G) * dim + (0 if values_are_keys else G * vdim), n_seq, max_q_len
    a.n_state, a.R = ring.shape[:2] if ring is not None else (n_slots, a.taps)
    if pooled is not None:
        table = meta["page_table"]
        a.pooled, a.page_table, a.pool, a.pool_rows, a.pool_stride, a.n_pooled, a.max_pages = ptr(pooled), ptr(table), pool, pooled_page_rows(pool), pooled.stride(0), pooled.shape[0], table.shape[1]
    if (w is not None and w.shape[1] != a.C) or (ring is not None and (ring.shape[2] != a.C or not ring.is_contiguous())):
        raise ValueError("conv_qkv: convolution weights, ring and heads differ in channels")
    call("cuteafd_conv_qkv", ctypes.addressof(a), _f32(proj), stream())


def pooled_page_rows(pool: int) -> int:
    """Pooled rows that belong to a page of 64 tokens: whole strips of eight blocks, each with the page of its first token."""
    return 8 * -(-8 // pool)


def pool_kv(cache, pooled, pool: int, page_table, kv_len, q_len, *, width: int, n_seq: int, max_q_len: int, status=None):
    """Means over blocks of `pool` cached rows (`width` elements each) for every block that a run of more than 16 tokens completes; `pooled`
    [pages * pooled_page_rows(pool), .] is addressed through the page table (see `csrc/attn_extras.cuh`)."""
    call("cuteafd_pool_kv", ptr(cache), cache.stride(0), cache.shape[0], ptr(pooled), pooled.stride(0), pooled.shape[0], width, pool, pooled_page_rows(pool), ptr(page_table),
         page_table.shape[1], ptr(kv_len), ptr(q_len), n_seq, max_q_len, _f32(cache), ptr(status), stream())


def recurrence_arg(x, y, x_b, y_b, conv, conv_b, ring, state, u, gates, gates_b, decay, agg, out, meta: dict, *, blocks, T, ldt, tiles, n_tiles, tn, n_seq, max_q_len,
                   status=None):
    """Arguments of one recurrent layer's step (`rglru_conv`, the gate product, `lru_scan`): x, y column views of one projection buffer; u block-major
    [blocks * ldt, n_pad]; `ring` [slots, depth + taps - 1, width], `state` [slots, depth + 1, width] by position."""
    a = native.Recurrence()
    for n, t in dict(x=x, y=y, x_b=x_b, y_b=y_b, conv=conv, conv_b=conv_b, ring=ring, state=state, u=u, gates=gates, gates_b=gates_b, decay=decay, agg=agg, out=out,
                     tiles=tiles, n_tiles=n_tiles, status=status, **{k: meta[k] for k in ("state_slot", "q_start", "q_len", "kv_len")}).items():
        setattr(a, n, ptr(t))
    a.n_state, a.depth, a.C = state.shape[0], state.shape[1] - 1, state.shape[2]
    a.taps, a.sq, a.sqp = conv.shape[0], a.C // blocks, u.shape[-1]
    if ring.shape != (a.n_state, a.taps - 1 + a.depth, a.C) or x.stride(0) != y.stride(0):
        raise ValueError("recurrence: ring, state and projection do not belong together")
    a.ldp, a.ldt, a.ldg, a.ldo, a.tn, a.T, a.n_seq, a.max_q_len = x.stride(0), ldt, gates.stride(0), out.stride(0), tn, T, n_seq, max_q_len
    a.agg_rows = agg.shape[0] if agg is not None else 0
    return a


def rglru_conv(a, *, f32: bool):
    call("cuteafd_rglru_conv", ctypes.addressof(a), 1 if f32 else 0, stream())


def lru_scan(a, *, f32: bool):
    call("cuteafd_lru_scan", ctypes.addressof(a), 1 if f32 else 0, stream())


def glu_rows(g, u, gate_b, up_b, out, rows: int, limit: float):
    """out = clamped GLU of two projected rows with biases (`tc_linear`'s clamped_glu epilogue as a pass of its own)."""
    call("cuteafd_glu_rows", ptr(g), ptr(u), ptr(gate_b), ptr(up_b), ptr(out), rows, g.stride(0), out.stride(0), g.shape[1], float(limit), _f32(g), stream())


def encode_window_maps(rows: torch.Tensor, Hkv: int, dp: int, dvp: int, box_rows: int = 64) -> torch.Tensor:
    """TMA descriptors (uint8 [2, 128]: keys, values) of one layer's store [slots, row]: Hkv key heads of dp elements, then Hkv value heads of dvp;
    `box_rows` 8: of its pooled blocks."""
    host = torch.zeros(2, 128, dtype=torch.uint8)
    call("cuteafd_tmap_encode_heads", host[0].data_ptr(), rows.data_ptr(), dp, Hkv, rows.stride(0), rows.shape[0], box_rows)
    call("cuteafd_tmap_encode_heads", host[1].data_ptr(), rows.data_ptr() + Hkv * dp * rows.element_size(), dvp, Hkv, rows.stride(0), rows.shape[0], box_rows)
    return host.to(rows.device)


def attn_extras(sink=None, gate=None, per_value: bool = False, keep_first: int = 0, out_scale: float = 1.0, pooled=None, pool_maps=None, pool: int = 0):
    """What an attention layer has besides: a `sink` logit per head (fp32 [Hq]); `gate` logits (column view of the projection rows: one per head, or
    `per_value` one per output value) whose sigmoid multiplies the output; the sequence's first `keep_first` keys visible behind the window; or one key
    and value for each block of `pool` tokens wholly in front of it (`pooled`: rows of the blocks, `pool_maps`: their descriptors); a constant factor
    on the output."""
    x = native.AttnExtras()
    x.sink, x.gate, x.ldg = ptr(sink), ptr(gate), gate.stride(0) if gate is not None else 0
    x.gate_values, x.keep_first, x.out_scale = 1 if per_value else 0, keep_first, float(out_scale)
    if pool:
        x.pooled, x.pool_maps, x.pool, x.pool_rows = ptr(pooled), ptr(pool_maps), pool, pooled_page_rows(pool)
    return x


def _extras(x):
    return ctypes.addressof(x) if x is not None else None


def window_attention(q, maps, page_table, kv_len, q_start, q_len, out, *, T, n_seq, max_q_len, Hq, Hkv, dp, dvp, dv, n_splits=1, part_o=None, part_ml=None, window=0, scale,
                     prefill=False, extras=None, status=None):
    """Windowed paged GQA on the tensor cores (key / value heads of their own, padded widths); `prefill`: the 128-key kernel (dp + 2 dvp <= 512);
    `extras`: see `attn_extras`."""
    head = (ptr(q), ptr(maps), ptr(page_table), ptr(kv_len), ptr(q_start), ptr(q_len), ptr(out))
    shape = (T, n_seq, max_q_len, q.stride(0), Hq, Hkv, dp, dvp, dv, out.stride(0), page_table.shape[1])
    if prefill:
        call("cuteafd_window_prefill_attention", *head, *shape, window, float(scale), _extras(extras), ptr(status), stream())
    else:
        call("cuteafd_window_attention", *head, ptr(part_o), ptr(part_ml), *shape, n_splits, window, float(scale), _extras(extras), ptr(status), stream())


def window_attention_simt(q, cache, page_table, kv_len, q_start, q_len, out, *, T, n_seq, Hq, Hkv, dp, dvp, dv, window=0, scale, extras=None, pool_stride=0, status=None):
    """The same on the ordinary cores: fp32, heads wider than 256, groups of more than 128; `pool_stride`: elements between two pooled rows."""
    call("cuteafd_window_attention_simt", ptr(q), q.stride(0), ptr(cache), ptr(page_table), ptr(kv_len), ptr(q_start), ptr(q_len), ptr(out), out.stride(0), T, n_seq, Hq,
         Hkv, dp, dvp, dv, cache.stride(0), pool_stride, page_table.shape[1], cache.shape[0], window, float(scale), _f32(q), _extras(extras), ptr(status), stream())


# ------------------------------------------------------------------ hyper-connected stacks: stream boundaries, linear attention with a decay
HYPER_EMBED, HYPER_ADD, HYPER_GATHER = 0, 1, 2
SCAN_CHUNK = 128            # tokens of a chunk of `decay_scan`'s long form


def hyper_rows(x, W: int, rows: int, *, f32: bool, eps: float, next_in=None, gain=None, xn=None, tokens=None, table=None, pairs=None, meta=None, n_seq: int = 0, out=None,
               mix=None, a=None, b=None, bias=None, norms=None, scales=(1.0, 1.0), routed=None, src_rows=None, status=None):
    """Residual streams x (fp32 [., S, Wp], norms average over W) at a sub-layer boundary.

    With `tokens`: every stream = table[token] + the pair table's row; `pairs` = (rows, mul_prev, mul_cur, recent): the row number is
    (previous token * mul_prev + token * mul_cur) mod buckets, the row behind the last starts a sequence; `recent` int32 [slots, R] keeps the
    tokens fed by position, `meta` and `n_seq` are the step's sequences.
    With `out` / `mix`: x_t = sum_s mix[s, t] x_s + out[t] y, where y = scales[0] * (a + bias) + scales[1] * b (with `norms` = two gains, each
    RMS-normed first) + the weighted rows of `routed` = (y, slot_row, wts, k).
    Otherwise the rows listed in `src_rows`, collapsed by summing the streams.
    `xn` receives the collapsed rows (weights `next_in`) RMS-normed with `gain`."""
    _chk(x, torch.float32, "x")
    r = native.HyperRows()
    r.x, r.S, r.W, r.Wp, r.eps, r.status = ptr(x), x.shape[1], W, x.shape[2], eps, ptr(status)
    r.next_in, r.gain, r.xn, r.ldn = ptr(next_in), ptr(gain), ptr(xn), xn.stride(0) if xn is not None else 0
    mode = HYPER_GATHER
    for t in (table, a, b):
        if t is not None and t.shape[1] != x.shape[2]:
            raise ValueError("hyper_rows: rows and residual streams differ in width")
    if tokens is not None:
        _chk(tokens, torch.int32, "tokens"); _chk(table, torch.bfloat16, "table")
        mode, r.tokens, r.table, r.vocab = HYPER_EMBED, ptr(tokens), ptr(table), table.shape[0]
        if pairs is not None:
            rows_, r.mul_prev, r.mul_cur, recent = pairs
            _chk(rows_, torch.bfloat16, "pairs"); _chk(recent, torch.int32, "recent")
            r.pair_rows, r.buckets, r.recent, r.R, r.n_seq, r.n_state = ptr(rows_), rows_.shape[0] - 1, ptr(recent), recent.shape[1], n_seq, recent.shape[0]
            for n in ("state_slot", "q_start", "q_len", "kv_len"):
                setattr(r, n, ptr(meta[n]))
    elif mix is not None:
        mode, r.out, r.mix, r.a, r.b, r.bias = HYPER_ADD, ptr(out), ptr(mix), ptr(a), ptr(b), ptr(bias)
        r.sa, r.sb = float(scales[0]), float(scales[1])
        if norms is not None:
            r.ga, r.gb = ptr(norms[0]), ptr(norms[1])
        if routed is not None:
            y, slot_row, wts, r.k = routed
            r.y, r.slot_row, r.wts = ptr(y), ptr(slot_row), ptr(wts)
    else:
        r.src_rows = ptr(src_rows)
    call("cuteafd_hyper_rows", ctypes.addressof(r), mode, rows, 1 if f32 else 0, stream())


def decay_scan_arg(q, k, v, g, state, tags, ring, out, meta: dict, *, H, dim, vdim, n_seq, max_q_len, eps, rope=None, pairs=0, q_scale=1.0, k_scale=1.0, decay=None, low_rank=None, forget=None,
                   tau=1.0, norm=None, out_scale=1.0, chunks=None, T: int = 0, status=None):
    """Arguments of `decay_scan`: q, k, v, g column views of one projection buffer; `decay` fp32 [H] (constant) or `low_rank` = (a1 column view, a2 fp32
    [H * dim, rank], bias fp32 [H * dim]): decay sigmoid(a2 a1 + bias) ** (1 / tau) per key channel, or `forget` = (bias, lower bound; fp32 [H * dim]):
    HGRN2, where k are the forget gate's logits and q passes SiLU; g None: no output gate; `state` [slots, 2, H, dim, vp] with `tags`
    [slots, H, 2] (positions), `ring` [slots, depth, H, 2 dim + vp].  `chunks`: scratch of `scan_scratch`, with which long runs of a step of
    `T` rows take the chunk kernels (bf16, heads of up to 128 x 256)."""
    a = native.DecayScan()
    if chunks is not None:
        a.chunk_state, a.chunk_decay, a.chunk_tiles, a.chunks, a.T = ptr(chunks[0]), ptr(chunks[1]), ptr(chunks[2]), chunks[0].shape[0], T
        if chunks[0].shape[1:] != (H, dim, state.shape[-1]) or any(c.shape[0] != a.chunks for c in chunks):
            raise ValueError("decay_scan: chunk scratch of another geometry")
    for n, t in dict(q=q, k=k, v=v, g=g, rope=rope, decay=decay, norm=norm, state=state, tags=tags, ring=ring, out=out, status=status,
                     **{m: meta[m] for m in ("state_slot", "q_start", "q_len", "kv_len")}).items():
        setattr(a, n, ptr(t))
    if low_rank is not None:
        a.a1, a.a2, a.a2_b, a.rank = ptr(low_rank[0]), ptr(low_rank[1]), ptr(low_rank[2]), low_rank[1].shape[1]
    if forget is not None:
        a.forget_b, a.lower = ptr(forget[0]), ptr(forget[1])
    if not q.stride(0) == k.stride(0) == v.stride(0) == (g.stride(0) if g is not None else v.stride(0)):
        raise ValueError("decay_scan: q, k, v and gate are columns of one buffer")
    a.ldp, a.pairs, a.ldo, a.H, a.dim, a.vdim, a.vp, a.depth, a.n_state = q.stride(0), pairs, out.stride(0), H, dim, vdim, state.shape[-1], ring.shape[1], state.shape[0]
    a.n_seq, a.max_q_len, a.q_scale, a.k_scale, a.inv_tau, a.eps, a.out_scale = n_seq, max_q_len, q_scale, k_scale, 1.0 / tau, eps, out_scale
    if state.shape[1:4] != (2, H, dim) or ring.shape[2:] != (H, 2 * dim + a.vp) or tags.shape != (a.n_state, H, 2):
        raise ValueError("decay_scan: state, tags and ring do not belong together")
    return a


def scan_scratch(rows: int, n_seq: int, H: int, dim: int, vdim: int, device) -> tuple:
    """Scratch of `decay_scan`'s chunk kernels for steps of up to `rows` rows of up to `n_seq` sequences (zeroed: pads of the operand tiles stay zero)."""
    n, up = rows // SCAN_CHUNK + n_seq + 1, lambda v, m: -(-v // m) * m
    return (torch.zeros(n, H, dim, up(vdim, 4), dtype=torch.float32, device=device), torch.zeros(n, H, 2 * dim + 1, dtype=torch.float32, device=device),
            torch.zeros(n, H, 2, up(dim, 64) * up(vdim, 64), dtype=torch.bfloat16, device=device))


def decay_scan(a, *, f32: bool):
    call("cuteafd_decay_scan", ctypes.addressof(a), 1 if f32 else 0, stream())


def side_gate(z, tokens, table, col: int, n: int, out, rows: int, *, status=None):
    """out[t, :n] = gelu_tanh(z[t, :n]) * table[token, col : col + n] (z fp32, the table bf16)."""
    _chk(z, torch.float32, "z"); _chk(tokens, torch.int32, "tokens"); _chk(table, torch.bfloat16, "table")
    call("cuteafd_side_gate", ptr(z), z.stride(0), ptr(tokens), ptr(table), table.stride(0), col, n, table.shape[0], ptr(out), out.stride(0), rows, _f32(out), ptr(status), stream())


def silu_rows(g, u, out, rows: int):
    """out = silu(g) * u over two projected rows (`tc_linear`'s SwiGLU epilogue as a pass of its own)."""
    call("cuteafd_silu_rows", ptr(g), ptr(u), ptr(out), rows, g.stride(0), out.stride(0), g.shape[1], _f32(g), stream())

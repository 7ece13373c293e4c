// MLA prefill attention on the 5th-generation tensor cores: the NON-absorbed form for long query chunks.
//
// Decode multiplies the query into the 512-wide latent space and attends over the latent cache (attention_mla.cu): per key
// that is 576 + 512 multiply-adds per head, fine while the step is bound by reading the cache.  A prefill chunk is bound by
// arithmetic, and the per-head form needs 192 + 128 multiply-adds per key: the latent rows of the sequence's context are
// first expanded once per chunk into per-head keys and values (one GEMM with the kv_b projection, `kvb` below), then
//   S[128 x 128] = [q_nope | q_rope] [k_nope | k_rope]^T      three 64-wide chunks, tcgen05.mma kind::f16, N = 128 keys
//   O[128 x 128] += softmax(S) V
// (a tcgen05.mma of M = 128 costs ~130 cycles whatever its N up to 256, so key tiles are 128 wide: 12 score + 8 PV
// instructions per 128 keys instead of 24 + 8 with 64-key tiles)
// with a CTA owning 128 query tokens of ONE head.  k_rope is shared by all heads and comes straight from the gathered latent
// rows (columns 512..575); k_nope and V come from the expanded buffer [rows, Hl * 256] (per head: 128 key columns, then 128
// value columns).  Both buffers are contiguous per sequence (`ctx_start[seq]` + key index), so tiles need no page table.
//
// Structure (one CTA per SM, 192 threads): warp 0 streams K tiles (48 KB, two stages) and V tiles (32 KB, two stages) by TMA;
// the 128 x 192 query tile sits in tensor memory (96 columns) as the A operand of the score MMAs, which leaves the shared
// memory to the K / V rings; warp 1 issues the MMAs (scores double-buffered in tensor memory), warps 2-5
// run the softmax, one thread per row in two passes over the tile's 128 score columns (maximum, then exponentials, which
// are computed BEFORE the wait for the PV product of tile i - 1, so that product runs under them).
// Every wait is bounded and reports through the status word.
//
// Reference: the dedicated MLA prefill kernels of the GLM5 family (native/families/glm5/cuda/glm_mla_prefill.cu:123, 539),
// which also expand the latent cache per chunk and run per-head attention with mma.sync.
#include <string.h>

#define CA_PDL_CLASS 2
#include "common.cuh"
#include "attn_extras.cuh"

#define PF_KT 128                 // keys per tile
#define PF_NS 2                   // K stages
#define PF_NSV 2                  // V stages
#define PF_Q_BYTES 0              // the query tile lives in tensor memory (A operand of the score MMAs)
#define PF_P_BYTES 32768          // 2 chunks (64 keys each) x [128 rows x 128 B]
#define PF_V_STAGE 32768          // 2 chunks (64 dims each) x [128 keys x 128 B]

struct MlaPrefillArgs {
  const bf16* q_nope;           // [Hl, T, 128] head-major
  const bf16* q_rope;           // rotated parts, 64 wide: row (t, head) at t * qr_t + head * qr_h
  const float* sink;            // [Hl], or null
  CUtensorMap kvb_map;          // {Hl * 256, rows, 1}, box {64, 128, 1}, 128-byte swizzle (encoded with rank 3: loads pass z = 0)
  CUtensorMap lat_map;          // {576, rows, 1}, box {64, 128, 1}, 128-byte swizzle
  const int* ctx_start;         // [n_seq] first row of the sequence's context in the two buffers
  const int* kv_len;
  const int* q_start;
  const int* q_len;
  const float* gate;            // [T, Hl] factor of each head's output, or null
  bf16* out;                    // [T, ldo] token-major, head h at column h * dv
  int* status;
  int T, Hl, max_q_tiles;
  int qr_t, qr_h, rope_col;     // (rope_col: column of the latent rows where the rotated key part starts)
  int ldt, ldo, dv;             // rows between two heads of q_nope, output row stride, value width
  float scale;
};

__device__ __forceinline__ uint64_t pf_desc_mn_sw128(uint32_t saddr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= (uint64_t)((saddr & 0x3FFFF) >> 4);
  d |= (uint64_t)(lbo >> 4) << 16;
  d |= (uint64_t)(sbo >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}
__device__ __forceinline__ uint32_t pf_idesc(int n, int b_mn_major) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)b_mn_major << 16) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
}
__device__ __forceinline__ void pf_tmem_st_x16(uint32_t addr, const uint32_t* r) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
               ::"r"(addr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]),
                 "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]) : "memory");
}

// KN 64-wide chunks of per-head key columns, KR rotated chunks shared by the heads (0 = attention without positions), NV chunks of value
// columns; the expanded buffer holds (KN + NV) * 64 columns per head.  DeepSeek-V3: 2, 1, 2.
template <int KN, int KR, int NV>
__global__ void __launch_bounds__(192, 1) mla_prefill_kernel(const __grid_constant__ MlaPrefillArgs a) {
  pdl_launch(); pdl_wait();
  constexpr int NK = KN + KR, K_STAGE = NK * 16384, V_STAGE = NV * 16384, HEAD_W = (KN + NV) * 64;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* sP = smem;
  uint8_t* sK = sP + PF_P_BYTES;
  uint8_t* sV = sK + PF_NS * K_STAGE;
  uint64_t* bars = (uint64_t*)(sV + PF_NSV * V_STAGE);
  uint64_t* k_full = bars; uint64_t* k_empty = bars + 2; uint64_t* v_full = bars + 4; uint64_t* v_empty = bars + 6;     // [<= 2] each
  uint64_t* s_full = bars + 8;          // [2]
  uint64_t* s_free = bars + 10;         // [2]: the softmax threads are done with the score buffer
  uint64_t& p_full = bars[12]; uint64_t& o_done = bars[13];
  uint32_t& tmem_slot = *(uint32_t*)(bars + 14);
  int& abort_flag = *(int*)(bars + 15);
  if (smem_u32(smem) & 1023) { if (threadIdx.x == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0xA13); return; }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;

  // the heaviest query tiles (most visible keys) are scheduled first
  const int head = blockIdx.x;
  const int seq = blockIdx.y / a.max_q_tiles, qt = a.max_q_tiles - 1 - blockIdx.y % a.max_q_tiles;
  const int qlen = a.q_len[seq], kvlen = a.kv_len[seq];
  const int tok0 = qt * 128;
  if (tok0 >= qlen) return;
  const int R = min(128, qlen - tok0);
  const int row_base = a.q_start[seq] + tok0;
  const int first_pos = kvlen - qlen + tok0;
  const int hi = first_pos + R;
  const int n_tiles = (hi + PF_KT - 1) / PF_KT;
  const int ctx0 = a.ctx_start[seq];

  if (tid == 0) {
    for (int s = 0; s < 2; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); }
    for (int s = 0; s < 2; ++s) { mbar_init(&s_full[s], 1); mbar_init(&s_free[s], 128); }
    mbar_init(&p_full, 128); mbar_init(&o_done, 1);
    abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 1) { tmem_alloc(&tmem_slot, 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  volatile int* abortp = &abort_flag;
  const uint32_t S0_COL = 0, O_COL = 128, S1_COL = 256, Q_COL = 384;
  // query rows -> tensor memory (row = lane, two bf16 per 32-bit column, 32 columns per 64-wide chunk: q_nope low / high, q_rope)
  if (warp >= 2) {
    const int r = (warp & 3) * 32 + lane;
    const uint32_t dst = tmem + ((uint32_t)((warp & 3) * 32) << 16) + Q_COL;
    const int t = row_base + (r < R ? r : 0);
    const bf16* src_nope = a.q_nope + ((size_t)head * a.ldt + t) * (KN * 64);
    const bf16* src_rope = a.q_rope + (size_t)t * a.qr_t + (size_t)head * a.qr_h;
#pragma unroll 1
    for (int g = 0; g < 2 * NK; ++g) {             // 16 columns = 32 elements per store
      const bf16* src = (KR == 0 || g < 2 * KN) ? src_nope + g * 32 : src_rope + (g - 2 * KN) * 32;
      uint32_t w[16];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const uint4 v = r < R ? *(const uint4*)(src + j * 8) : make_uint4(0, 0, 0, 0);
        w[4 * j] = v.x; w[4 * j + 1] = v.y; w[4 * j + 2] = v.z; w[4 * j + 3] = v.w;
      }
      pf_tmem_st_x16(dst + g * 16, w);
    }
    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();

  if (warp == 0) {
    // ------------------------------------------------------------------ K / V producer
    // K runs one tile ahead of V in this warp's program order: the single V stage only frees when the previous PV product
    // retires, and the K tile of the NEXT score pass must not queue behind that wait.
    auto load_k = [&](int i) -> bool {
      const int s = i % PF_NS, ph = ((i / PF_NS) & 1) ^ 1;
      if (!mbar_wait_bounded(&k_empty[s], ph, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_PRODUCER, i); return false; }
      if (lane == 0) {
        const int row = ctx0 + i * PF_KT;
        mbar_expect_tx(&k_full[s], K_STAGE);
#pragma unroll
        for (int c = 0; c < KN; ++c) tma_load_3d(sK + s * K_STAGE + c * 16384, &a.kvb_map, &k_full[s], head * HEAD_W + c * 64, row, 0);
        if (KR) tma_load_3d(sK + s * K_STAGE + KN * 16384, &a.lat_map, &k_full[s], a.rope_col, row, 0);
      }
      __syncwarp();
      return true;
    };
    bool okp = n_tiles > 0 ? load_k(0) : true;
    for (int i = 0; okp && i < n_tiles && !*abortp; ++i) {
      if (i + 1 < n_tiles && !load_k(i + 1)) break;
      const int sv = i % PF_NSV, phv = ((i / PF_NSV) & 1) ^ 1;
      if (!mbar_wait_bounded(&v_empty[sv], phv, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_PRODUCER, 0x1000 + i); break; }
      if (lane == 0) {
        const int row = ctx0 + i * PF_KT;
        mbar_expect_tx(&v_full[sv], V_STAGE);
#pragma unroll
        for (int c = 0; c < NV; ++c) tma_load_3d(sV + sv * V_STAGE + c * 16384, &a.kvb_map, &v_full[sv], head * HEAD_W + (KN + c) * 64, row, 0);
      }
      __syncwarp();
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    const uint32_t id_s = pf_idesc(PF_KT, 0), id_o = pf_idesc(NV * 64, 1);
    auto issue_scores = [&](int j) -> bool {     // S[j & 1] = Q K(j)^T once the softmax threads have copied tile j - 2 out of it
      const int s = j % PF_NS;
      if (j >= 2 && !mbar_wait_bounded(&s_free[j & 1], ((j - 2) >> 1) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_MMA, 0x2000 + j); return false; }
      if (!mbar_wait_bounded(&k_full[s], (j / PF_NS) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_MMA, j); return false; }
      tc_fence_after();
      if (lane == 0) {
        const uint32_t k0 = smem_u32(sK + s * K_STAGE), d = tmem + ((j & 1) ? S1_COL : S0_COL);
#pragma unroll
        for (int kb = 0; kb < NK; ++kb)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            tc_mma_f16_ta(d, tmem + Q_COL + kb * 32 + k * 8, umma_desc_sw128(k0 + kb * 16384) + 2 * k, id_s, (kb | k) ? 1u : 0u);
        tc_commit(&s_full[j & 1]);
        tc_commit(&k_empty[s]);
      }
      __syncwarp();
      return true;
    };
    bool ok = true;
    for (int j = 0; ok && j < min(2, n_tiles); ++j) ok = issue_scores(j);
    for (int i = 0; ok && i < n_tiles; ++i) {
      const int sv = i % PF_NSV;
      if (!mbar_wait_bounded(&p_full, i & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_MMA, 0x3000 + i); break; }
      if (!mbar_wait_bounded(&v_full[sv], (i / PF_NSV) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_MMA, 0x4000 + i); break; }
      tc_fence_after();
      if (lane == 0) {
        const uint32_t v0 = smem_u32(sV + sv * V_STAGE);
#pragma unroll
        for (int k = 0; k < PF_KT / 16; ++k)       // 16 keys per MMA: P chunk k / 4 (64 keys per 128-byte row), V rows 16 k .. 16 k + 15
          tc_mma_f16(tmem + O_COL, umma_desc_sw128(smem_u32(sP) + (k >> 2) * 16384) + 2 * (k & 3), pf_desc_mn_sw128(v0 + k * 2048, 16384, 1024), id_o,
                     (i | k) ? 1u : 0u);
        tc_commit(&v_empty[sv]);
        tc_commit(&o_done);
      }
      __syncwarp();
      if (i + 2 < n_tiles) ok = issue_scores(i + 2);
    }
  } else {
    // ------------------------------------------------------------------ softmax + epilogue: thread = query row
    const int q4 = warp & 3, r = q4 * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(q4 * 32) << 16;
    const bool live = r < R;
    const int qpos = live ? first_pos + r : -1;
    const float sc2 = a.scale * 1.4426950408889634f;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    for (int i = 0; i < n_tiles; ++i) {
      if (!mbar_wait_bounded(&s_full[i & 1], (i >> 1) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_EPILOGUE, i); ok = false; break; }
      tc_fence_after();
      const uint32_t s_addr = tmem + lane_addr + ((i & 1) ? S1_COL : S0_COL);
      const int key0 = i * PF_KT;
      const bool all_visible = key0 + PF_KT - 1 <= first_pos;      // CTA-uniform: every key of the tile is visible to every live row
      // two passes over the tile's 128 score columns: row maximum, then exponentials packed to bf16 pairs (64 registers).
      // Tiles below the diagonal need no mask (CTA-uniform test), which is all but the last one or two of a long context.
      float mx = -INFINITY;
      uint32_t pk[PF_KT / 2];
      float psum = 0.f;
      float alpha = 1.f;
      if (all_visible) {           // CTA-uniform (the tensor-memory loads below are warp collectives); rows past R hold zero queries
#pragma unroll 1
        for (int c = 0; c < PF_KT / 32; ++c) {
          uint32_t sr[32];
          tmem_ld_x16(s_addr + c * 32, sr);
          tmem_ld_x16(s_addr + c * 32 + 16, sr + 16);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) mx = fmaxf(mx, __uint_as_float(sr[j]));
        }
        mx *= sc2;                                   // sc2 > 0: scaling commutes with the maximum
        if (mx > m_ref + 8.f) {
          if (m_ref != -INFINITY) { alpha = exp2f(m_ref - mx); l *= alpha; }
          m_ref = mx;
        }
#pragma unroll
        for (int c = 0; c < PF_KT / 32; ++c) {
          uint32_t sr[32];
          tmem_ld_x16(s_addr + c * 32, sr);
          tmem_ld_x16(s_addr + c * 32 + 16, sr + 16);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float e0 = exp2f(fmaf(__uint_as_float(sr[2 * j]), sc2, -m_ref)), e1 = exp2f(fmaf(__uint_as_float(sr[2 * j + 1]), sc2, -m_ref));
            psum += e0 + e1;
            bf162 h = __floats2bfloat162_rn(e0, e1);
            pk[c * 16 + j] = *(uint32_t*)&h;
          }
        }
      } else {
#pragma unroll 1
        for (int c = 0; c < PF_KT / 32; ++c) {
          uint32_t sr[32];
          tmem_ld_x16(s_addr + c * 32, sr);
          tmem_ld_x16(s_addr + c * 32 + 16, sr + 16);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            const int kp = key0 + c * 32 + j;
            if (live && kp <= qpos) mx = fmaxf(mx, __uint_as_float(sr[j]) * sc2);
          }
        }
        if (mx > m_ref + 8.f) {
          if (m_ref != -INFINITY) { alpha = exp2f(m_ref - mx); l *= alpha; }
          m_ref = mx;
        }
#pragma unroll
        for (int c = 0; c < PF_KT / 32; ++c) {
          uint32_t sr[32];
          tmem_ld_x16(s_addr + c * 32, sr);
          tmem_ld_x16(s_addr + c * 32 + 16, sr + 16);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const int kp = key0 + c * 32 + 2 * j;
            const float e0 = (live && kp <= qpos) ? exp2f(fmaf(__uint_as_float(sr[2 * j]), sc2, -m_ref)) : 0.f;
            const float e1 = (live && kp + 1 <= qpos) ? exp2f(fmaf(__uint_as_float(sr[2 * j + 1]), sc2, -m_ref)) : 0.f;
            psum += e0 + e1;
            bf162 h = __floats2bfloat162_rn(e0, e1);
            pk[c * 16 + j] = *(uint32_t*)&h;
          }
        }
      }
      l += psum;
      tc_fence_before();
      mbar_arrive(&s_free[i & 1]);
      // the previous P V product must have finished before P is overwritten or O rescaled
      if (i > 0 && !mbar_wait_bounded(&o_done, (i - 1) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_EPILOGUE, 0x1000 + i); ok = false; break; }
      tc_fence_after();
      if (i > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {      // warp-uniform: tcgen05.ld/st are warp collectives
#pragma unroll 1
        for (int c = 0; c < NV * 4; ++c) {
          uint32_t o[16];
          tmem_ld_x16(tmem + lane_addr + O_COL + c * 16, o);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
          pf_tmem_st_x16(tmem + lane_addr + O_COL + c * 16, o);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      }
      // P: two K-major chunks of 64 keys; 16-byte unit u of a row holds keys 8 u .. 8 u + 7
#pragma unroll
      for (int u = 0; u < PF_KT / 8; ++u)
        *(uint4*)(sP + (u >> 3) * 16384 + r * 128 + (((u & 7) ^ (r & 7)) << 4)) = make_uint4(pk[4 * u], pk[4 * u + 1], pk[4 * u + 2], pk[4 * u + 3]);
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(&p_full);
    }
    if (ok && n_tiles > 0 && !mbar_wait_bounded(&o_done, (n_tiles - 1) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_EPILOGUE, 999); ok = false; }
    tc_fence_after();
    if (__all_sync(0xffffffffu, ok)) {
      const int t = row_base + (live ? r : 0);
      float scale_o = 1.f, lt = l;
      if (a.sink) {                                     // learned sink logit: one more softmax term with a zero value
        const float m_nat = (m_ref == -INFINITY) ? -INFINITY : m_ref * 0.6931471805599453f, sk = a.sink[head], m2 = fmaxf(m_nat, sk);
        const float e1 = (m_nat == -INFINITY) ? 0.f : __expf(m_nat - m2);
        lt = l * e1 + __expf(sk - m2); scale_o = e1;
      }
      const float inv = (lt > 0.f ? scale_o / lt : 0.f) * ((a.gate && live) ? a.gate[(size_t)t * a.Hl + head] : 1.f);      // output gate of the head
      bf16* dst = a.out + (size_t)t * a.ldo + (size_t)head * a.dv;
      const bool vec = (a.ldo | a.dv) % 8 == 0;
#pragma unroll 1
      for (int c = 0; c < NV * 4; ++c) {
        uint32_t o[16];
        if (n_tiles > 0) { tmem_ld_x16(tmem + lane_addr + O_COL + c * 16, o); tc_wait_ld(); }
        else {
#pragma unroll
          for (int j = 0; j < 16; ++j) o[j] = 0;
        }
        if (!live) continue;
        uint32_t w[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) { bf162 hh = __floats2bfloat162_rn(__uint_as_float(o[2 * j]) * inv, __uint_as_float(o[2 * j + 1]) * inv); w[j] = *(uint32_t*)&hh; }
        if (vec) {                            // value widths that do not fill their last 64-wide chunk stop at column dv
          if (c * 16 < a.dv) *(uint4*)(dst + c * 16) = make_uint4(w[0], w[1], w[2], w[3]);
          if (c * 16 + 8 < a.dv) *(uint4*)(dst + c * 16 + 8) = make_uint4(w[4], w[5], w[6], w[7]);
        } else {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (c * 16 + j < a.dv) dst[c * 16 + j] = ((const bf16*)w)[j];
        }
      }
    }
  }
  if (*abortp && warp == 0) { const uint64_t t0 = globaltimer_ns(); while (globaltimer_ns() - t0 < 200000) __nanosleep(1000); }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, 512);
}

// ------------------------------------------------------------------------------------------------------------
// The same structure for paged GQA prefill, templated on the 64-wide chunks of key (KC) and value (VC) dimensions (head_dim 128: 2, 2): a CTA owns 128 query rows of one KV head (row = token_in_tile * G +
// head_in_group) and walks the sequence's pages two at a time (128-key tiles), K and V straight from the paged store.  Causal
// mask, optional sliding window and sink logit as in the decode kernel (attention_tc.cu), no split-KV: a prefill chunk has
// enough query tiles to fill the GPU.  window < 0 drops the causal mask (bidirectional attention of a vision / audio encoder:
// every query row sees keys [0, kvlen)).  The 64-key decode kernel spends 8 + 4 tcgen05.mma per 64 keys; this one 8 + 8 per 128 keys.
template <int KC, int VC>
struct GqaPrefillCfg {
  static constexpr int K_STAGE = KC * 16384, V_STAGE = VC * 16384;          // chunks (64 dims each) x [128 keys x 128 B]
  static constexpr int NSV = PF_P_BYTES + PF_NS * K_STAGE + 2 * V_STAGE <= 224 * 1024 ? 2 : 1;
  static constexpr int SMEM = PF_P_BYTES + PF_NS * K_STAGE + NSV * V_STAGE + 256;
  static_assert(256 + KC * 32 + VC * 64 <= 512, "scores, query and output exceed tensor memory");
};
struct GqaPrefillArgs {
  const bf16* q;
  const CUtensorMap* k_map; const CUtensorMap* v_map;      // the decode kernel's descriptors; value head h at coordinate v_head0 + h
  const int* page_table; const int* kv_len; const int* q_start; const int* q_len;
  AttnExtras<bf16> x;                                      // sink, kept first keys, output gate
  bf16* out;
  int* status;
  int q_stride, Hq, Hkv, max_pages, window, max_q_tiles;
  int v_head0, dv, ldo;
  float scale;
};

template <int KC, int VC>
__global__ void __launch_bounds__(192, 1) gqa_prefill_kernel(const __grid_constant__ GqaPrefillArgs a) {
  using Cf = GqaPrefillCfg<KC, VC>;
  pdl_launch(); pdl_wait();
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* sP = smem;
  uint8_t* sK = sP + PF_P_BYTES;
  uint8_t* sV = sK + PF_NS * Cf::K_STAGE;
  uint64_t* bars = (uint64_t*)(sV + Cf::NSV * Cf::V_STAGE);
  uint64_t* k_full = bars; uint64_t* k_empty = bars + 2; uint64_t* v_full = bars + 4; uint64_t* v_empty = bars + 6;     // [<= 2] each
  uint64_t* s_full = bars + 8;          // [2]
  uint64_t* s_free = bars + 10;         // [2]: the softmax threads are done with the score buffer
  uint64_t& p_full = bars[12]; uint64_t& o_done = bars[13];
  uint32_t& tmem_slot = *(uint32_t*)(bars + 14);
  int& abort_flag = *(int*)(bars + 15);
  if (smem_u32(smem) & 1023) { if (threadIdx.x == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0xA14); return; }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;

  // the heaviest query tiles (most visible keys) are scheduled first
  const int G = a.Hq / a.Hkv, tok_per_tile = 128 / G;
  const int kvh = blockIdx.x;
  const int seq = blockIdx.y / a.max_q_tiles, qt = a.max_q_tiles - 1 - blockIdx.y % a.max_q_tiles;
  const int qlen = a.q_len[seq], kvlen = a.kv_len[seq];
  const int tok0 = qt * tok_per_tile;
  if (tok0 >= qlen) return;
  const int ntok = min(tok_per_tile, qlen - tok0);
  const int R = ntok * G;                                   // row = token_in_tile * G + head_in_group
  const int row_base = a.q_start[seq] + tok0;
  const bool bidir = a.window < 0;                          // encoder towers: every row sees all kvlen keys
  const int first_pos = bidir ? kvlen - 1 : kvlen - qlen + tok0;
  const int hi = bidir ? kvlen : first_pos + ntok;
  const int lo = a.window > 0 ? max(0, first_pos - a.window + 1) : 0;
  const int tile0 = lo / PF_KT;
  // tiles of kept first keys or of pooled blocks in front of the window, then the window's
  const int kept = a.x.lead_tiles(tile0, PF_KT, hi - 1, a.window), n_tiles = kept + max(0, (hi + PF_KT - 1) / PF_KT - tile0);
  auto tile_at = [&](int i) { return i < kept ? i : i - kept + tile0; };
  auto pooled_at = [&](int i) { return a.x.pool > 0 && i < kept; };

  if (tid == 0) {
    for (int s = 0; s < 2; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); }
    for (int s = 0; s < 2; ++s) { mbar_init(&s_full[s], 1); mbar_init(&s_free[s], 128); }
    mbar_init(&p_full, 128); mbar_init(&o_done, 1);
    abort_flag = 0;
    fence_barrier_init();
  }
  if (warp == 1) { tmem_alloc(&tmem_slot, 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  volatile int* abortp = &abort_flag;
  const uint32_t S0_COL = 0, S1_COL = 128, O_COL = 256, Q_COL = 256 + VC * 64;
  // query rows -> tensor memory (row = lane, two bf16 per 32-bit column, 32 columns per chunk)
  if (warp >= 2) {
    const int r = (warp & 3) * 32 + lane;
    const uint32_t dst = tmem + ((uint32_t)((warp & 3) * 32) << 16) + Q_COL;
    const int rr = r < R ? r : 0;
    const bf16* src = a.q + (size_t)(row_base + rr / G) * a.q_stride + (size_t)(kvh * G + rr % G) * (KC * 64);
#pragma unroll 1
    for (int g = 0; g < KC * 2; ++g) {                  // 16 columns = 32 elements per store
      uint32_t w[16];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const uint4 v = r < R ? *(const uint4*)(src + g * 32 + j * 8) : make_uint4(0, 0, 0, 0);
        w[4 * j] = v.x; w[4 * j + 1] = v.y; w[4 * j + 2] = v.z; w[4 * j + 3] = v.w;
      }
      pf_tmem_st_x16(dst + g * 16, w);
    }
    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();

  if (warp == 0) {
    // ------------------------------------------------------------------ K / V producer
    // K runs one tile ahead of V in this warp's program order: the single V stage only frees when the previous PV product
    // retires, and the K tile of the NEXT score pass must not queue behind that wait.
    auto page_of = [&](int key) -> int {                   // pages past the sequence's table are read as page 0 (finite rows, masked keys)
      const int pi = key / 64;
      return pi < a.max_pages ? a.page_table[(size_t)seq * a.max_pages + pi] : 0;
    };
    // lane l's strip of a tile of pooled blocks (past the last one: that one again, masked)
    auto strip_of = [&](int i) { return a.x.strip_row(min(tile_at(i) * 16 + (lane & 15), (a.x.blocks_seen(hi - 1, a.window) - 1) >> 3), a.page_table + (size_t)seq * a.max_pages); };
    auto load_k = [&](int i) -> bool {
      const int s = i % PF_NS, ph = ((i / PF_NS) & 1) ^ 1;
      if (!mbar_wait_bounded(&k_empty[s], ph, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_PRODUCER, i); return false; }
      if (pooled_at(i)) {
        const int row = strip_of(i);
        if (lane == 0) mbar_expect_tx(&k_full[s], Cf::K_STAGE);
        __syncwarp();
        if (lane < 16) {
#pragma unroll
          for (int c = 0; c < KC; ++c) tma_load_3d(sK + s * Cf::K_STAGE + c * 16384 + lane * 1024, a.x.pool_maps, &k_full[s], c * 64, kvh, row);
        }
      } else if (lane == 0) {
        const int key0 = tile_at(i) * PF_KT;
        mbar_expect_tx(&k_full[s], Cf::K_STAGE);
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          const int slot0 = page_of(key0 + p * 64) * 64;
#pragma unroll
          for (int c = 0; c < KC; ++c) tma_load_3d(sK + s * Cf::K_STAGE + c * 16384 + p * 8192, a.k_map, &k_full[s], c * 64, kvh, slot0);
        }
      }
      __syncwarp();
      return true;
    };
    bool okp = n_tiles > 0 ? load_k(0) : true;
    for (int i = 0; okp && i < n_tiles && !*abortp; ++i) {
      if (i + 1 < n_tiles && !load_k(i + 1)) break;
      const int sv = i % Cf::NSV, phv = ((i / Cf::NSV) & 1) ^ 1;
      if (!mbar_wait_bounded(&v_empty[sv], phv, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_PRODUCER, 0x1000 + i); break; }
      if (pooled_at(i)) {
        const int row = strip_of(i);
        if (lane == 0) mbar_expect_tx(&v_full[sv], Cf::V_STAGE);
        __syncwarp();
        if (lane < 16) {
#pragma unroll
          for (int c = 0; c < VC; ++c) tma_load_3d(sV + sv * Cf::V_STAGE + c * 16384 + lane * 1024, a.x.pool_maps + 1, &v_full[sv], c * 64, kvh, row);
        }
      } else if (lane == 0) {
        const int key0 = tile_at(i) * PF_KT;
        mbar_expect_tx(&v_full[sv], Cf::V_STAGE);
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          const int slot0 = page_of(key0 + p * 64) * 64;
#pragma unroll
          for (int c = 0; c < VC; ++c) tma_load_3d(sV + sv * Cf::V_STAGE + c * 16384 + p * 8192, a.v_map, &v_full[sv], c * 64, a.v_head0 + kvh, slot0);
        }
      }
      __syncwarp();
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    const uint32_t id_s = pf_idesc(PF_KT, 0), id_o = pf_idesc(VC * 64, 1);
    auto issue_scores = [&](int j) -> bool {     // S[j & 1] = Q K(j)^T once the softmax threads have copied tile j - 2 out of it
      const int s = j % PF_NS;
      if (j >= 2 && !mbar_wait_bounded(&s_free[j & 1], ((j - 2) >> 1) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_MMA, 0x2000 + j); return false; }
      if (!mbar_wait_bounded(&k_full[s], (j / PF_NS) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_MMA, j); return false; }
      tc_fence_after();
      if (lane == 0) {
        const uint32_t k0 = smem_u32(sK + s * Cf::K_STAGE), d = tmem + ((j & 1) ? S1_COL : S0_COL);
#pragma unroll
        for (int kb = 0; kb < KC; ++kb)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            tc_mma_f16_ta(d, tmem + Q_COL + kb * 32 + k * 8, umma_desc_sw128(k0 + kb * 16384) + 2 * k, id_s, (kb | k) ? 1u : 0u);
        tc_commit(&s_full[j & 1]);
        tc_commit(&k_empty[s]);
      }
      __syncwarp();
      return true;
    };
    bool ok = true;
    for (int j = 0; ok && j < min(2, n_tiles); ++j) ok = issue_scores(j);
    for (int i = 0; ok && i < n_tiles; ++i) {
      const int sv = i % Cf::NSV;
      if (!mbar_wait_bounded(&p_full, i & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_MMA, 0x3000 + i); break; }
      if (!mbar_wait_bounded(&v_full[sv], (i / Cf::NSV) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_MMA, 0x4000 + i); break; }
      tc_fence_after();
      if (lane == 0) {
        const uint32_t v0 = smem_u32(sV + sv * Cf::V_STAGE);
#pragma unroll
        for (int k = 0; k < PF_KT / 16; ++k)       // 16 keys per MMA: P chunk k / 4 (64 keys per 128-byte row), V rows 16 k .. 16 k + 15
          tc_mma_f16(tmem + O_COL, umma_desc_sw128(smem_u32(sP) + (k >> 2) * 16384) + 2 * (k & 3), pf_desc_mn_sw128(v0 + k * 2048, 16384, 1024), id_o,
                     (i | k) ? 1u : 0u);
        tc_commit(&v_empty[sv]);
        tc_commit(&o_done);
      }
      __syncwarp();
      if (i + 2 < n_tiles) ok = issue_scores(i + 2);
    }
  } else {
    // ------------------------------------------------------------------ softmax + epilogue: thread = query row
    const int q4 = warp & 3, r = q4 * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(q4 * 32) << 16;
    const bool live = r < R;
    const int qpos = live ? (bidir ? first_pos : first_pos + r / G) : -1;
    const int wlo = a.window > 0 ? qpos - a.window : -1;           // keys at or below this position are outside the row's window
    const int blocks = live ? a.x.blocks_seen(qpos, a.window) : 0;
    const float sc2 = a.scale * 1.4426950408889634f;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    for (int i = 0; i < n_tiles; ++i) {
      if (!mbar_wait_bounded(&s_full[i & 1], (i >> 1) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_EPILOGUE, i); ok = false; break; }
      tc_fence_after();
      const uint32_t s_addr = tmem + lane_addr + ((i & 1) ? S1_COL : S0_COL);
      const int key0 = tile_at(i) * PF_KT;
      // CTA-uniform: every key of the tile is visible to every live row (below the diagonal and inside every row's window)
      // (tiles of pooled blocks: of the blocks that a row sees)
      const bool pooled = pooled_at(i);
      const bool all_visible = pooled ? key0 + PF_KT <= a.x.blocks_seen(first_pos, a.window)
                                      : key0 + PF_KT - 1 <= first_pos && (a.window <= 0 || key0 > first_pos + ntok - 1 - a.window || key0 + PF_KT <= a.x.keep_first);
      auto sees = [&](int kp) { return pooled ? kp < blocks : live && kp <= qpos && (kp > wlo || kp < a.x.keep_first); };
      // two passes over the tile's 128 score columns: row maximum, then exponentials packed to bf16 pairs (64 registers).
      // Tiles below the diagonal need no mask (CTA-uniform test), which is all but the last one or two of a long context.
      float mx = -INFINITY;
      uint32_t pk[PF_KT / 2];
      float psum = 0.f;
      float alpha = 1.f;
      if (all_visible) {           // CTA-uniform (the tensor-memory loads below are warp collectives); rows past R hold zero queries
#pragma unroll 1
        for (int c = 0; c < PF_KT / 32; ++c) {
          uint32_t sr[32];
          tmem_ld_x16(s_addr + c * 32, sr);
          tmem_ld_x16(s_addr + c * 32 + 16, sr + 16);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) mx = fmaxf(mx, __uint_as_float(sr[j]));
        }
        mx *= sc2;                                   // sc2 > 0: scaling commutes with the maximum
        if (mx > m_ref + 8.f) {
          if (m_ref != -INFINITY) { alpha = exp2f(m_ref - mx); l *= alpha; }
          m_ref = mx;
        }
#pragma unroll
        for (int c = 0; c < PF_KT / 32; ++c) {
          uint32_t sr[32];
          tmem_ld_x16(s_addr + c * 32, sr);
          tmem_ld_x16(s_addr + c * 32 + 16, sr + 16);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float e0 = exp2f(fmaf(__uint_as_float(sr[2 * j]), sc2, -m_ref)), e1 = exp2f(fmaf(__uint_as_float(sr[2 * j + 1]), sc2, -m_ref));
            psum += e0 + e1;
            bf162 h = __floats2bfloat162_rn(e0, e1);
            pk[c * 16 + j] = *(uint32_t*)&h;
          }
        }
      } else {
#pragma unroll 1
        for (int c = 0; c < PF_KT / 32; ++c) {
          uint32_t sr[32];
          tmem_ld_x16(s_addr + c * 32, sr);
          tmem_ld_x16(s_addr + c * 32 + 16, sr + 16);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            const int kp = key0 + c * 32 + j;
            if (sees(kp)) mx = fmaxf(mx, __uint_as_float(sr[j]) * sc2);
          }
        }
        if (mx > m_ref + 8.f) {
          if (m_ref != -INFINITY) { alpha = exp2f(m_ref - mx); l *= alpha; }
          m_ref = mx;
        }
#pragma unroll
        for (int c = 0; c < PF_KT / 32; ++c) {
          uint32_t sr[32];
          tmem_ld_x16(s_addr + c * 32, sr);
          tmem_ld_x16(s_addr + c * 32 + 16, sr + 16);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const int kp = key0 + c * 32 + 2 * j;
            const float e0 = sees(kp) ? exp2f(fmaf(__uint_as_float(sr[2 * j]), sc2, -m_ref)) : 0.f;
            const float e1 = sees(kp + 1) ? exp2f(fmaf(__uint_as_float(sr[2 * j + 1]), sc2, -m_ref)) : 0.f;
            psum += e0 + e1;
            bf162 h = __floats2bfloat162_rn(e0, e1);
            pk[c * 16 + j] = *(uint32_t*)&h;
          }
        }
      }
      l += psum;
      tc_fence_before();
      mbar_arrive(&s_free[i & 1]);
      // the previous P V product must have finished before P is overwritten or O rescaled
      if (i > 0 && !mbar_wait_bounded(&o_done, (i - 1) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_EPILOGUE, 0x1000 + i); ok = false; break; }
      tc_fence_after();
      if (i > 0 && __any_sync(0xffffffffu, alpha != 1.f)) {      // warp-uniform: tcgen05.ld/st are warp collectives
#pragma unroll 1
        for (int c = 0; c < VC * 4; ++c) {
          uint32_t o[16];
          tmem_ld_x16(tmem + lane_addr + O_COL + c * 16, o);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
          pf_tmem_st_x16(tmem + lane_addr + O_COL + c * 16, o);
        }
        asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      }
      // P: two K-major chunks of 64 keys; 16-byte unit u of a row holds keys 8 u .. 8 u + 7
#pragma unroll
      for (int u = 0; u < PF_KT / 8; ++u)
        *(uint4*)(sP + (u >> 3) * 16384 + r * 128 + (((u & 7) ^ (r & 7)) << 4)) = make_uint4(pk[4 * u], pk[4 * u + 1], pk[4 * u + 2], pk[4 * u + 3]);
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(&p_full);
    }
    if (ok && n_tiles > 0 && !mbar_wait_bounded(&o_done, (n_tiles - 1) & 1, abortp)) { ca_dev_fail(a.status, CA_DEV_TIMEOUT_EPILOGUE, 999); ok = false; }
    tc_fence_after();
    if (__all_sync(0xffffffffu, ok)) {
      const int rr = live ? r : 0;
      const int t = row_base + rr / G, h = kvh * G + rr % G;
      float scale_o = 1.f, lt = l;
      if (a.x.sink) {                                   // learned sink logit: one more softmax term with a zero value
        const float m_nat = (m_ref == -INFINITY) ? -INFINITY : m_ref * 0.6931471805599453f;
        const float sk = a.x.sink[h], m2 = fmaxf(m_nat, sk);
        const float e1 = (m_nat == -INFINITY) ? 0.f : __expf(m_nat - m2);
        lt = l * e1 + __expf(sk - m2); scale_o = e1;
      }
      const float inv = (lt > 0.f ? scale_o / lt : 0.f) * a.x.head_factor(t, h);
      const bool gated = a.x.gate && a.x.gate_values;
      bf16* dst = a.out + (size_t)t * a.ldo + (size_t)h * a.dv;
      const bool vec = ((a.dv | a.ldo) & 7) == 0;
#pragma unroll 1
      for (int c = 0; c < VC * 4; ++c) {
        uint32_t o[16];
        if (n_tiles > 0) { tmem_ld_x16(tmem + lane_addr + O_COL + c * 16, o); tc_wait_ld(); }
        else {
#pragma unroll
          for (int j = 0; j < 16; ++j) o[j] = 0;
        }
        if (!live) continue;
        if (gated) {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (c * 16 + j < a.dv) o[j] = __float_as_uint(__uint_as_float(o[j]) * a.x.value_factor(t, h * a.dv + c * 16 + j));
        }
        uint32_t w[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) { bf162 hh = __floats2bfloat162_rn(__uint_as_float(o[2 * j]) * inv, __uint_as_float(o[2 * j + 1]) * inv); w[j] = *(uint32_t*)&hh; }
        if (vec) {
          if (c * 16 < a.dv) *(uint4*)(dst + c * 16) = make_uint4(w[0], w[1], w[2], w[3]);
          if (c * 16 + 8 < a.dv) *(uint4*)(dst + c * 16 + 8) = make_uint4(w[4], w[5], w[6], w[7]);
        } else {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (c * 16 + j < a.dv) dst[c * 16 + j] = ((const bf16*)w)[j];
        }
      }
    }
  }
  if (*abortp && warp == 0) { const uint64_t t0 = globaltimer_ns(); while (globaltimer_ns() - t0 < 200000) __nanosleep(1000); }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, 512);
}

template <int KC, int VC>
static int launch_gqa_prefill(const GqaPrefillArgs& a, int n_seq, cudaStream_t s) {
  const int smem = GqaPrefillCfg<KC, VC>::SMEM;
  static bool attr_set[64] = {false};
  int dev = 0; cudaGetDevice(&dev);
  if (!attr_set[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(gqa_prefill_kernel<KC, VC>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return ca_cuda(e, "cudaFuncSetAttribute(gqa_prefill)");
    attr_set[dev & 63] = true;
  }
  CA_LAUNCH_PDL((gqa_prefill_kernel<KC, VC>), dim3(a.Hkv, n_seq * a.max_q_tiles), 192, smem, s, a);
  CA_CHECK_LAUNCH("gqa_prefill_attention");
  return CA_OK;
}

extern "C" int cuteafd_gqa_prefill_attention(const void* q, const void* kv_map, const int* page_table, const int* kv_len, const int* q_start,
                                             const int* q_len, const float* sink, void* out, int T, int n_seq, int max_q_len, int q_stride, int Hq,
                                             int Hkv, int max_pages, int window, float scale, int* status, cudaStream_t s) {
  CA_REQUIRE(q && kv_map && page_table && kv_len && q_start && q_len && out, "gqa_prefill_attention: null argument");
  CA_REQUIRE(Hq % Hkv == 0 && 128 % (Hq / Hkv) == 0 && q_stride % 8 == 0, "gqa_prefill_attention: group size %d unsupported", Hq / Hkv);
  if (T <= 0 || n_seq <= 0) return CA_OK;
  GqaPrefillArgs a;
  a.q = (const bf16*)q; a.k_map = a.v_map = (const CUtensorMap*)kv_map; a.v_head0 = Hkv; a.dv = 128; a.ldo = Hq * 128; a.page_table = page_table; a.kv_len = kv_len; a.q_start = q_start; a.q_len = q_len;
  a.x = attn_extras<bf16>(nullptr, 0); a.x.sink = sink; a.out = (bf16*)out; a.status = status; a.q_stride = q_stride; a.Hq = Hq; a.Hkv = Hkv; a.max_pages = max_pages; a.window = window;
  a.scale = scale;
  const int tpt = 128 / (Hq / Hkv);
  a.max_q_tiles = (max_q_len + tpt - 1) / tpt;
  return launch_gqa_prefill<2, 2>(a, n_seq, s);
}

// The same over a store whose keys and values have widths of their own (layout and maps as `cuteafd_window_attention`); dk_pad + 2 dv_pad
// of at most 512 fit tensor memory.
extern "C" int cuteafd_window_prefill_attention(const void* q, const void* maps, const int* page_table, const int* kv_len, const int* q_start, const int* q_len, void* out,
                                                int T, int n_seq, int max_q_len, int q_stride, int Hq, int Hkv, int dk_pad, int dv_pad, int dv, int ldo, int max_pages,
                                                int window, float scale, const CaAttnExtras* extras, int* status, cudaStream_t s) {
  CA_REQUIRE(q && maps && page_table && kv_len && q_start && q_len && out, "window_prefill_attention: null argument");
  CA_REQUIRE(Hkv >= 1 && Hq % Hkv == 0 && Hq / Hkv <= 128 && q_stride % 8 == 0, "window_prefill_attention: group size %d unsupported", Hkv ? Hq / Hkv : 0);
  CA_REQUIRE(dv >= 1 && dv <= dv_pad && ldo >= Hq * dv && window >= 0 && q_stride >= Hq * dk_pad, "window_prefill_attention: bad shape");
  CA_REQUIRE(!extras || !extras->gate || extras->ldg >= (extras->gate_values ? Hq * dv : Hq), "window_prefill_attention: gate rows too short");
  CA_REQUIRE(attn_extras_ok(extras, true), "window_prefill_attention: pooled blocks without their rows, or beside kept keys");
  if (T <= 0 || n_seq <= 0) return CA_OK;
  GqaPrefillArgs a = {};
  a.q = (const bf16*)q; a.k_map = (const CUtensorMap*)maps; a.v_map = a.k_map + 1; a.v_head0 = 0; a.page_table = page_table; a.kv_len = kv_len; a.q_start = q_start;
  a.q_len = q_len; a.x = attn_extras<bf16>(extras, window); a.out = (bf16*)out; a.status = status; a.q_stride = q_stride; a.Hq = Hq; a.Hkv = Hkv; a.max_pages = max_pages; a.window = window;
  a.scale = scale; a.dv = dv; a.ldo = ldo;
  const int tpt = 128 / (Hq / Hkv);
  a.max_q_tiles = (max_q_len + tpt - 1) / tpt;
#define WP_CASE(K_, V_) if (dk_pad == K_ * 64 && dv_pad == V_ * 64) return launch_gqa_prefill<K_, V_>(a, n_seq, s);
  WP_CASE(1, 1) WP_CASE(1, 2) WP_CASE(1, 3) WP_CASE(2, 1) WP_CASE(2, 2) WP_CASE(2, 3) WP_CASE(3, 1) WP_CASE(3, 2) WP_CASE(4, 1) WP_CASE(4, 2)
  return ca_fail(CA_ERR_UNSUPPORTED, "window_prefill_attention: head widths %d / %d do not fit tensor memory", dk_pad, dv_pad);
}

// Gathers the latent rows of every sequence's context out of the paged cache into one contiguous buffer:
// dst[ctx_start[s] + j] = cache[page_table[s][j / 64] * 64 + j % 64] for j < kv_len[s]; rows of w16 16-byte pieces (72: 576 bf16),
// src16 pieces between two rows of the cache; a block copies blockDim / w16 rows.
__global__ void mla_gather_ctx_kernel(const uint4* __restrict__ cache, const int* __restrict__ page_table, const int* __restrict__ ctx_start,
                                      const int* __restrict__ kv_len, uint4* __restrict__ dst, int max_pages, long long n_slots, long long dst_rows, int w16,
                                      int src16, int* status) {
  pdl_launch(); pdl_wait();
  const int seq = blockIdx.y;
  const int j = blockIdx.x * (blockDim.x / w16) + threadIdx.x / w16, c = threadIdx.x % w16;
  if (j >= kv_len[seq]) return;
  const long long slot = (long long)page_table[(size_t)seq * max_pages + j / 64] * 64 + j % 64;
  const long long row = (long long)ctx_start[seq] + j;
  if (slot < 0 || slot >= n_slots || row < 0 || row >= dst_rows) { if (c == 0) ca_dev_fail(status, CA_DEV_BAD_INDEX, 0xB01); return; }
  dst[row * w16 + c] = cache[slot * src16 + c];
}

extern "C" int cuteafd_mla_gather_ctx(const void* cache, const int* page_table, const int* ctx_start, const int* kv_len, void* dst, int n_seq,
                                      int max_kv, int max_pages, long long n_slots, long long dst_rows, int* status, cudaStream_t s) {
  CA_REQUIRE(cache && page_table && ctx_start && kv_len && dst, "mla_gather_ctx: null argument");
  if (n_seq <= 0 || max_kv <= 0) return CA_OK;
  CA_LAUNCH_PDL(mla_gather_ctx_kernel, dim3((max_kv + 3) / 4, n_seq), 288, 0, s, (const uint4*)cache, page_table, ctx_start, kv_len, (uint4*)dst, max_pages,
                n_slots, dst_rows, 72, 72, status);
  CA_CHECK_LAUNCH("mla_gather_ctx");
  return CA_OK;
}

// Rows of `width` bf16 (a multiple of 8, at most 4096) out of a cache whose rows are `row_stride` apart.
extern "C" int cuteafd_latent_gather_ctx(const void* cache, const int* page_table, const int* ctx_start, const int* kv_len, void* dst, int n_seq,
                                         int max_kv, int max_pages, long long n_slots, long long dst_rows, int width, int row_stride, int* status,
                                         cudaStream_t s) {
  CA_REQUIRE(cache && page_table && ctx_start && kv_len && dst, "latent_gather_ctx: null argument");
  CA_REQUIRE(width % 8 == 0 && width >= 8 && width <= 4096 && row_stride % 8 == 0 && width <= row_stride, "latent_gather_ctx: bad row width %d / %d", width, row_stride);
  if (n_seq <= 0 || max_kv <= 0) return CA_OK;
  const int w16 = width / 8, rpb = w16 >= 256 ? 1 : 256 / w16;
  CA_LAUNCH_PDL(mla_gather_ctx_kernel, dim3((max_kv + rpb - 1) / rpb, n_seq), w16 * rpb, 0, s, (const uint4*)cache, page_table, ctx_start, kv_len,
                (uint4*)dst, max_pages, n_slots, dst_rows, w16, row_stride / 8, status);
  CA_CHECK_LAUNCH("latent_gather_ctx");
  return CA_OK;
}

template <int KN, int KR, int NV>
static int mla_prefill_launch(const MlaPrefillArgs& a, int n_seq, cudaStream_t s) {
  constexpr int SMEM = PF_P_BYTES + PF_NS * (KN + KR) * 16384 + PF_NSV * NV * 16384 + 256;
  auto kern = mla_prefill_kernel<KN, KR, NV>;
  static bool attr_set[64] = {false};
  int dev = 0; cudaGetDevice(&dev);
  if (!attr_set[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
    if (e != cudaSuccess) return ca_cuda(e, "cudaFuncSetAttribute(mla_prefill)");
    attr_set[dev & 63] = true;
  }
  CA_LAUNCH_PDL(kern, dim3(a.Hl, n_seq * a.max_q_tiles), 192, SMEM, s, a);
  return CA_OK;
}

// q_nope [Hl, T, 128] (head-major), q_rope [T, Hl, 64], kvb [rows, Hl * 256], lat [rows, 576], out [T, Hl * 128].
extern "C" int cuteafd_mla_prefill_attention(const void* q_nope, const void* q_rope, const void* kvb, const void* lat, long long rows, const int* ctx_start,
                                             const int* kv_len, const int* q_start, const int* q_len, void* out, int T, int n_seq, int max_q_len, int Hl,
                                             float scale, int* status, cudaStream_t s) {
  CA_REQUIRE(q_nope && q_rope && kvb && lat && out && rows > 0, "mla_prefill_attention: null argument");
  CA_REQUIRE(Hl >= 1, "mla_prefill_attention: no heads");
  if (T <= 0 || n_seq <= 0) return CA_OK;
  MlaPrefillArgs a;
  int rc = ca_encode_tmap_2d(&a.kvb_map, kvb, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (uint64_t)Hl * 256, (uint64_t)rows, (uint64_t)Hl * 512, 64, PF_KT,
                             CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  rc = ca_encode_tmap_2d(&a.lat_map, lat, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 576, (uint64_t)rows, 1152, 64, PF_KT, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  a.q_nope = (const bf16*)q_nope; a.q_rope = (const bf16*)q_rope; a.ctx_start = ctx_start; a.kv_len = kv_len; a.q_start = q_start; a.q_len = q_len;
  a.out = (bf16*)out; a.status = status; a.T = T; a.Hl = Hl; a.max_q_tiles = (max_q_len + 127) / 128; a.scale = scale;
  a.gate = nullptr; a.ldt = T; a.ldo = Hl * 128; a.dv = 128; a.sink = nullptr; a.qr_t = Hl * 64; a.qr_h = 64; a.rope_col = 512;
  rc = mla_prefill_launch<2, 1, 2>(a, n_seq, s);
  if (rc) return rc;
  CA_CHECK_LAUNCH("mla_prefill_attention");
  return CA_OK;
}

// The same for latent attention of other sizes: q [Hl, ldt, dk_pad] head-major (dk_pad 64 / 128 / 192, pad columns zero), kvb
// [rows, Hl * (dk_pad + dv_pad)] (per head the key columns, then the value columns, each padded to whole 64-wide chunks; dv_pad 64 / 128),
// out [T, ldo] token-major with head h at column h * dv, `gate` [T, Hl] (or null) multiplied into each head's output, `sink` [Hl] (or null) one more
// logit per head.  With a rotated part (q_rope, null: attention without positions) of up to 64 dimensions: q_rope [Hl, ldt, 64] and, in the
// gathered context rows `lat` [rows, lat_width], 64 columns from `rope_col` on, shared by the heads; pad columns of q_rope are zero.
extern "C" int cuteafd_latent_prefill_attention(const void* q, const void* q_rope, const void* kvb, const void* lat, int lat_width, int rope_col, const float* sink, long long rows, const int* ctx_start, const int* kv_len,
                                                const int* q_start, const int* q_len, const float* gate, void* out, int T, int ldt, int n_seq,
                                                int max_q_len, int Hl, int dk_pad, int dv_pad, int dv, int ldo, float scale, int* status,
                                                cudaStream_t s) {
  CA_REQUIRE(q && kvb && ctx_start && kv_len && q_start && q_len && out && rows > 0, "latent_prefill_attention: null argument");
  CA_REQUIRE(Hl >= 1 && ldt >= T && dv >= 1 && dv <= dv_pad && ldo >= Hl * dv, "latent_prefill_attention: bad shape");
  CA_REQUIRE(!q_rope || (lat && rope_col % 64 == 0 && rope_col + 64 <= lat_width && lat_width % 8 == 0), "latent_prefill_attention: rotated part outside the context rows");
  CA_REQUIRE((dk_pad == 64 || dk_pad == 128 || dk_pad == 192) && (dv_pad == 64 || dv_pad == 128), "latent_prefill_attention: head widths %d / %d", dk_pad, dv_pad);
  if (T <= 0 || n_seq <= 0) return CA_OK;
  MlaPrefillArgs a;
  const int hw = dk_pad + dv_pad;
  int rc = ca_encode_tmap_2d(&a.kvb_map, kvb, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (uint64_t)Hl * hw, (uint64_t)rows, (uint64_t)Hl * hw * 2, 64, PF_KT,
                             CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  a.lat_map = a.kvb_map;
  if (q_rope) {
    rc = ca_encode_tmap_2d(&a.lat_map, lat, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (uint64_t)lat_width, (uint64_t)rows, (uint64_t)lat_width * 2, 64, PF_KT, CU_TENSOR_MAP_SWIZZLE_128B);
    if (rc) return rc;
  }
  a.sink = sink; a.qr_t = 64; a.qr_h = ldt * 64; a.rope_col = rope_col;
  a.q_nope = (const bf16*)q; a.q_rope = (const bf16*)q_rope; a.ctx_start = ctx_start; a.kv_len = kv_len; a.q_start = q_start; a.q_len = q_len;
  a.gate = gate; a.out = (bf16*)out; a.status = status; a.T = T; a.Hl = Hl; a.max_q_tiles = (max_q_len + 127) / 128; a.scale = scale;
  a.ldt = ldt; a.ldo = ldo; a.dv = dv;
#define LP_CASE(K_, R_, V_) if (dk_pad == K_ * 64 && dv_pad == V_ * 64 && (q_rope != nullptr) == (R_ != 0)) rc = mla_prefill_launch<K_, R_, V_>(a, n_seq, s);
#define LP_ROW(R_, V_) LP_CASE(1, R_, V_) LP_CASE(2, R_, V_) LP_CASE(3, R_, V_)
  LP_ROW(0, 1) LP_ROW(0, 2) LP_ROW(1, 1) LP_ROW(1, 2)
  if (rc) return rc;
  CA_CHECK_LAUNCH("latent_prefill_attention");
  return CA_OK;
}

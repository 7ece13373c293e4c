// Kernels of the hybrid recurrent / windowed-attention stacks (fp32 residual rows, RMS norms in front of and behind every sub-layer):
//   norm_rows        embedding, residual += mult * norm(sub-layer output + bias) (+ the embedding row once more), or a gather of rows - each also
//                    leaves the next product's operand row, normalised or as it is
//   rope_table       cosine / sine of the step's positions, once per rotation
//   conv_qkv         projected queries, keys and values (+ bias) -> short causal convolution -> norm (per head, over the whole projection, or
//                    none) -> rotation (neighbouring or half-apart pairs) -> query rows, paged cache; values may be the keys in front of the norm;
//                    short runs also leave the blocks they complete as pooled rows
//   pool_kv          cached rows -> means of the blocks that a long run completes
//   rglru_conv       x branch -> short causal convolution -> block-major operand of the gate product (and its tile table)
//   lru_scan         the real-gated linear recurrence: one pass over short runs, chunk aggregates + carried rescan over long ones
//   glu_rows         clamped GLU over two projected rows (all-fp32 mode; bf16 products do it in their epilogue)
//   window_attn_simt paged grouped-query attention on the ordinary cores (fp32, and shapes the tcgen05 kernels do not take): windows with kept
//                    first keys or pooled blocks, sinks, output gates
// Everything a sequence carries from step to step is addressed by absolute position: convolution inputs live in a ring of
// taps - 1 + depth rows, recurrent states in a ring of depth + 1, so a step that is repeated, or the last `depth` tokens that are taken back
// (rejected drafts), need no restore - later positions overwrite them.  T is the operand type: bf16, or float for the all-fp32 mode.
// (No counterpart in the reference, which has no such family; the recurrence's kernel is the sibling of linear_attn.cu.)
#include "stack_rows.cuh"
#include "attn_extras.cuh"

#define HS_TILE 16          // tokens of a sequence one block of the convolution kernels walks (at least taps - 1)
#define HS_MAX_TAPS 16
#define HS_CHUNK 64         // tokens of a chunk of the recurrence

// ---------------------------------------------------------------- residual rows and their norms
enum { ROWS_EMBED = 0, ROWS_ADD = 1, ROWS_GATHER = 2 };

template <typename T>
struct NormRows {
  float* x; int W, Wp;                                      // residual rows, Wp apart; norms average over W
  const int* tokens; const bf16* table; int vocab; float scale;        // ROWS_EMBED: scale times the token's row (ROWS_ADD with a table: added behind the rest)
  const T* add; const float* bias; const float* post; float mult;      // ROWS_ADD: bias and post (gain of the norm behind) may be null
  const int* src_rows;                                      // ROWS_GATHER
  const float* gain; T* xn; int ldn;                        // next operand: rows normalised by `gain` (null: without gains), or null
  int raw;                                                  // next operand: the rows as they are
  float eps; int* status;
};

template <typename T, int NCH, int MODE>
__global__ void norm_rows_kernel(const NormRows<T> a) {
  pdl_launch(); pdl_wait();
  __shared__ float red[32];
  const int t = blockIdx.x, nt = blockDim.x;
  float v[NCH][8];
  size_t row = t;
  if (MODE == ROWS_GATHER) row = (size_t)a.src_rows[t];
  int tok = 0;
  if (MODE == ROWS_EMBED || (MODE == ROWS_ADD && a.table)) {
    tok = a.tokens[t];
    if (tok < 0 || tok >= a.vocab) { if (threadIdx.x == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, t); tok = 0; }
  }
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * nt) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[c][j] = 0.f;
    if (i >= a.Wp) continue;
    if (MODE == ROWS_EMBED) {
      load8<bf16>(a.table + (size_t)tok * a.Wp + i, v[c]);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[c][j] *= a.scale;
    } else load8<float>(a.x + row * a.Wp + i, v[c]);
  }
  if (MODE == ROWS_ADD) {
    float m[NCH][8], ss = 0.f;
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
      const int i = (threadIdx.x + c * nt) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) m[c][j] = 0.f;
      if (i >= a.Wp) continue;
      load8<T>(a.add + (size_t)t * a.Wp + i, m[c]);
      if (a.bias) {
        float b[8];
        load8<float>(a.bias + i, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) m[c][j] += b[j];
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(m[c][j], m[c][j], ss);
    }
    const float inv = a.post ? rsqrtf(block_sum(ss, red) / (float)a.W + a.eps) : 1.f;
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
      const int i = (threadIdx.x + c * nt) * 8;
      if (i >= a.Wp) continue;
      float g[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
      if (a.post) load8<float>(a.post + i, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[c][j] = fmaf(a.mult, m[c][j] * inv * g[j], v[c][j]);
      if (a.table) {
        float e[8];
        load8<bf16>(a.table + (size_t)tok * a.Wp + i, e);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[c][j] = fmaf(a.scale, e[j], v[c][j]);
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * nt) * 8;
    if (i >= a.Wp) continue;
    if (MODE != ROWS_GATHER) store8<float>(a.x + (size_t)t * a.Wp + i, v[c]);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(v[c][j], v[c][j], ss);
  }
  if (!a.xn) return;
  const float inv = a.raw ? 1.f : rsqrtf(block_sum(ss, red) / (float)a.W + a.eps);
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * nt) * 8;
    if (i >= a.Wp) continue;
    float g[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f}, y[8];
    if (a.gain) load8<float>(a.gain + i, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) y[j] = v[c][j] * inv * g[j];
    store8<T>(a.xn + (size_t)t * a.ldn + i, y);
  }
}

// ---------------------------------------------------------------- rotation
// freq: [2, pairs] - the fp32 angle per position and what fp32 rounded off it, so that angles of far positions keep full accuracy.
__global__ void rope_table_kernel(const int* __restrict__ positions, const float* __restrict__ freq, float amp, int pairs, float2* __restrict__ out) {
  pdl_launch(); pdl_wait();
  const int t = blockIdx.x;
  const float p = (float)positions[t];
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
    const float f = freq[i], a = p * f, lo = fmaf(p, f, -a) + p * freq[pairs + i];
    float s, c;
    sincosf(a, &s, &c);
    const float cl = fmaf(-0.5f * lo, lo, 1.f), sl = lo * fmaf(lo * lo, -1.f / 6.f, 1.f);      // lo is at most half an ulp of a
    out[(size_t)t * pairs + i] = make_float2(amp * (c * cl - s * sl), amp * (s * cl + c * sl));
  }
}

// ---------------------------------------------------------------- short convolution in front of attention
enum { QK_NORM_NONE = 0, QK_NORM_HEAD = 1, QK_NORM_WHOLE = 2 };

template <typename T>
struct ConvQkv {
  const T* proj; int ldp;                       // [T, ldp]: H * dim queries | G * dim keys | G * vdim values (none with v_from_k)
  const float* w;                               // [taps, C]; null with one tap: no convolution
  const float* bias;                            // [C] of the projection, or null
  const float* q_norm; const float* k_norm;     // gains: [dim] of the head norms, [H * dim] and [G * dim] of the whole ones; null: none.  (A norm without
                                                // gains is the same in front of the rotation and behind it: rotations keep a head's sum of squares.)
  const float2* rope;                           // [T, pairs]
  T* ring;                                      // [slots, R, C] projected rows (without bias) by position; null with one tap
  const int* state_slot; const int* q_start; const int* q_len; const int* kv_len; const int* slot_map;
  T* q; int q_stride;                           // [T, H * dp]
  T* cache; int row_stride, n_slots;            // paged rows: G * dp keys, then G * dvp values
  int H, G, dim, dp, vdim, dvp, pairs, taps, R, C, n_state, norm, v_from_k;
  float eps; int* status;
  AttnExtras<T> pool;                           // blocks of pooled tokens (0: none); rows of `pooled` pool_stride apart
  T* pooled; const int* page_table; int max_pages, pool_stride, n_pooled;
};

template <typename T, int V> __device__ __forceinline__ void load_v(const T* p, float* v) {
  if constexpr (V == 8) {
    load8<T>(p, v);
  } else if constexpr (V == 4 && sizeof(T) == 2) {
    const uint2 q = *(const uint2*)p;
    const float2 x = __bfloat1622float2(*(const bf162*)&q.x), y = __bfloat1622float2(*(const bf162*)&q.y);
    v[0] = x.x; v[1] = x.y; v[2] = y.x; v[3] = y.y;
  } else if constexpr (V == 4) {
    const float4 q = *(const float4*)p;
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  } else if constexpr (V == 2 && sizeof(T) == 2) {
    const float2 x = __bfloat1622float2(*(const bf162*)p);
    v[0] = x.x; v[1] = x.y;
  } else if constexpr (V == 2) {
    const float2 x = *(const float2*)p;
    v[0] = x.x; v[1] = x.y;
  } else {
    v[0] = to_f(p[0]);
  }
}
template <typename T, int V> __device__ __forceinline__ void store_v(T* p, const float* v) {
  if constexpr (V == 8) {
    store8<T>(p, v);
  } else if constexpr (V == 4 && sizeof(T) == 2) {
    const bf162 x = __floats2bfloat162_rn(v[0], v[1]), y = __floats2bfloat162_rn(v[2], v[3]);
    *(uint2*)p = make_uint2(*(const uint32_t*)&x, *(const uint32_t*)&y);
  } else if constexpr (V == 4) {
    *(float4*)p = make_float4(v[0], v[1], v[2], v[3]);
  } else if constexpr (V == 2 && sizeof(T) == 2) {
    *(bf162*)p = __floats2bfloat162_rn(v[0], v[1]);
  } else if constexpr (V == 2) {
    *(float2*)p = make_float2(v[0], v[1]);
  } else {
    p[0] = to_t<T>(v[0]);
  }
}
// The first n of V elements (the others read as zero, or stay), with one access where `vec` says that all are there and aligned.
template <typename T, int V> __device__ __forceinline__ void load_n(const T* p, int n, bool vec, float* v) {
  if (vec) { load_v<T, V>(p, v); return; }
#pragma unroll
  for (int k = 0; k < V; ++k) v[k] = k < n ? to_f(p[k]) : 0.f;
}
template <typename T, int V> __device__ __forceinline__ void store_n(T* p, int n, bool vec, const float* v) {
  if (vec) { store_v<T, V>(p, v); return; }
#pragma unroll
  for (int k = 0; k < V; ++k) if (k < n) p[k] = to_t<T>(v[k]);
}

// One warp takes one head of a tile of HS_TILE tokens; a lane owns V neighbouring dimensions of the head (whole rotated pairs when neighbours
// turn together; with HALF the partner is half a rotation away and comes through `xch`).  TAPS > 0: the last inputs and the weights stay in
// registers; 0: any number of taps, inputs re-read.  STATS: only the sums of squares of the tile's rows, left in stats[i - i0]; otherwise
// `inv` holds the tile's factors of a norm over the whole projection (null: the norm is per head, or there is none).
template <typename T, int V, int TAPS, bool HALF, bool STATS>
__device__ __forceinline__ void conv_qkv_tile(const ConvQkv<T>& a, int unit, int seq, int i0, int i1, int slot, float* xch, float* stats, const float* inv) {
  const int lane = threadIdx.x & 31, n = a.q_len[seq], row0 = a.q_start[seq], p0 = a.kv_len[seq] - n;
  const bool is_q = unit < a.H, is_v = unit >= a.H + a.G;
  const int d = is_v ? a.vdim : a.dim, head = is_q ? unit : (is_v ? unit - a.H - a.G : unit - a.H), e = lane * V;
  const int ch = (is_v ? (a.H + a.G) * a.dim + head * a.vdim : unit * a.dim) + e;
  const int taps = TAPS ? TAPS : a.taps, own = max(0, min(V, d - e));      // dimensions of this lane
  const bool vec = own == V && ch % V == 0 && a.ldp % V == 0, wvec = own == V && ch % V == 0 && a.C % V == 0;
  T* ring = a.ring ? a.ring + (size_t)slot * a.R * a.C + ch : nullptr;
  float bias[V];
#pragma unroll
  for (int k = 0; k < V; ++k) bias[k] = a.bias && k < own ? a.bias[ch + k] : 0.f;
  // input row i of this run (i < 0: what the sequence fed before, nothing in front of its start)
  auto fresh = [&](int i, float* v) { load_n<T, V>(a.proj + (size_t)(row0 + i) * a.ldp + ch, own, vec, v); };
  auto input = [&](int i, float* v) {
    const int pos = p0 + i;
    if (i >= 0) fresh(i, v);
    else load_n<T, V>(ring + (size_t)((pos + a.R) % a.R) * a.C, pos < 0 ? 0 : own, pos >= 0 && wvec, v);
    if (pos >= 0)
#pragma unroll
      for (int k = 0; k < V; ++k) v[k] += bias[k];
  };
  auto weight = [&](int j, float* v) { load_n<float, V>(a.w + (size_t)j * a.C + ch, own, wvec, v); };
  constexpr int NH = TAPS > 1 ? TAPS - 1 : 1, NW = TAPS ? TAPS : 1;
  float hist[NH][V], wr[NW][V], gain[V];
  const float* gains = is_q ? a.q_norm : a.k_norm;
  const float* norm = gains + (a.norm == QK_NORM_WHOLE ? head * a.dim : 0);
#pragma unroll
  for (int k = 0; k < V; ++k) gain[k] = is_v || a.norm == QK_NORM_NONE || !gains ? 1.f : (k < own ? norm[e + k] : 0.f);
  if (TAPS) {
#pragma unroll
    for (int j = 0; j < NW; ++j) {
      if (a.w) weight(j, wr[j]);
      else
#pragma unroll
        for (int k = 0; k < V; ++k) wr[j][k] = 1.f;
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) input(i0 - (TAPS - 1) + j, hist[j]);
  }
  const bool keep = ring && n <= a.R - (taps - 1);      // short runs leave every input (a single tile), long ones the last taps - 1
  for (int i = i0; i < i1; ++i) {
    const int row = row0 + i;
    float cur[V], y[V], ss = 0.f;
    fresh(i, cur);
    constexpr int NT = HALF ? V : V / 2;
    float2 turn[NT];
    if (!STATS)
#pragma unroll
      for (int k = 0; k < NT; ++k) {
        const int pr = HALF ? (e + k < a.pairs ? e + k : e + k - a.pairs) : e / 2 + k;
        turn[k] = !is_v && pr < a.pairs ? a.rope[(size_t)row * a.pairs + pr] : make_float2(1.f, 0.f);
      }
    if (!STATS && keep && own) store_n<T, V>(ring + (size_t)((p0 + i) % a.R) * a.C, own, wvec, cur);
#pragma unroll
    for (int k = 0; k < V; ++k) { y[k] = 0.f; cur[k] += bias[k]; }
    if (TAPS) {
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] = fmaf(wr[j][k], hist[j][k], y[k]);
#pragma unroll
      for (int k = 0; k < V; ++k) y[k] = fmaf(wr[NW - 1][k], cur[k], y[k]);
#pragma unroll
      for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
        for (int k = 0; k < V; ++k) hist[j][k] = hist[j + 1][k];
      if (TAPS > 1)
#pragma unroll
        for (int k = 0; k < V; ++k) hist[NH - 1][k] = cur[k];
    } else {
      for (int j = 0; j < taps; ++j) {
        float u[V], w[V];
        input(i - (taps - 1) + j, u);
        weight(j, w);
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] = fmaf(w[k], u[k], y[k]);
      }
    }
#pragma unroll
    for (int k = 0; k < V; ++k) ss = fmaf(y[k], y[k], ss);
    if (STATS) {
      ss = warp_sum(ss);
      if (lane == 0) stats[i - i0] += ss;
      continue;
    }
    T* dst;
    if (is_q) dst = a.q + (size_t)row * a.q_stride + (size_t)head * a.dp;
    else {
      const int cs = a.slot_map[row];
      if (cs < 0 || cs >= a.n_slots) { if (lane == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, row); continue; }     // warp-uniform
      T* line = a.cache + (size_t)cs * a.row_stride;
      dst = line + (is_v ? (size_t)a.G * a.dp + (size_t)head * a.dvp : (size_t)head * a.dp);
      if (!is_v && a.v_from_k && own) store_n<T, V>(line + (size_t)a.G * a.dp + (size_t)head * a.dvp + e, own, own == V, y);
    }
    if (!is_v) {
      const float f = inv ? inv[i - i0] : (a.norm == QK_NORM_HEAD ? rsqrtf(warp_sum(ss) / (float)d + a.eps) : 1.f);
#pragma unroll
      for (int k = 0; k < V; ++k) y[k] *= f * gain[k];
      if constexpr (HALF) {
        if (a.pairs) {
#pragma unroll
          for (int k = 0; k < V; ++k) xch[e + k] = y[k];
          __syncwarp();
#pragma unroll
          for (int k = 0; k < V; ++k) {
            const int j = e + k;
            if (j < a.pairs) y[k] = y[k] * turn[k].x - xch[j + a.pairs] * turn[k].y;
            else if (j < 2 * a.pairs) y[k] = y[k] * turn[k].x + xch[j - a.pairs] * turn[k].y;
          }
          __syncwarp();
        }
      } else {
#pragma unroll
        for (int k = 0; k < V / 2; ++k) {
          const float u = y[2 * k], v = y[2 * k + 1];
          y[2 * k] = u * turn[k].x - v * turn[k].y; y[2 * k + 1] = v * turn[k].x + u * turn[k].y;
        }
      }
    }
    if (own) store_n<T, V>(dst + e, own, own == V, y);          // head starts are multiples of 64 elements
    if (!STATS && a.pooled && !is_q && own && n <= HS_TILE && (p0 + i + 1) % a.pool.pool == 0) {
      // the run is one tile: the block's rows are this lane's own, or of earlier steps
      const int P = a.pool.pool, b = (p0 + i) / P, *table = a.page_table + (size_t)seq * a.max_pages;
      const size_t off = (is_v ? (size_t)a.G * a.dp + (size_t)head * a.dvp : (size_t)head * a.dp) + e;
      const int row_b = a.pool.strip_row(b >> 3, table) + (b & 7);
      float m[V];
#pragma unroll
      for (int k = 0; k < V; ++k) m[k] = 0.f;
      bool ok = row_b >= 0 && row_b < a.n_pooled;
      for (int p = b * P; p < (b + 1) * P && ok; ++p) {
        const int cs = table[p / 64] * 64 + p % 64;
        if (cs < 0 || cs >= a.n_slots) { ok = false; break; }
        float u[V];
        load_n<T, V>(a.cache + (size_t)cs * a.row_stride + off, own, own == V, u);
#pragma unroll
        for (int k = 0; k < V; ++k) m[k] += u[k];
      }
      if (!ok) { ca_dev_fail(a.status, CA_DEV_BAD_INDEX, row); continue; }
#pragma unroll
      for (int k = 0; k < V; ++k) m[k] /= (float)P;
      store_n<T, V>(a.pooled + (size_t)row_b * a.pool_stride + off, own, own == V, m);
    }
  }
  if (!STATS && ring && !keep && i0 == 0 && own)          // this block read the old ring rows of these channels above: it may overwrite them now
    for (int i = max(0, n - (taps - 1)); i < n; ++i) {
      float v[V];
      fresh(i, v);
      store_n<T, V>(ring + (size_t)((p0 + i) % a.R) * a.C, own, wvec, v);
    }
}

// Norms per head (or none): a warp per (head, tile).  WHOLE: a block per tile, its warps share the heads out - sums of squares first, then
// everything else with the convolution once more (inputs are in L1).
#define HS_WHOLE_WARPS 16
template <typename T, int V, int TAPS, bool HALF, bool WHOLE>
__global__ void __launch_bounds__(WHOLE ? HS_WHOLE_WARPS * 32 : 128) conv_qkv_kernel(const ConvQkv<T> a) {
  pdl_launch(); pdl_wait();
  constexpr int NWARP = WHOLE ? HS_WHOLE_WARPS : 4;
  __shared__ float xch[HALF ? NWARP : 1][HALF ? 32 * V : 1];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, seq = blockIdx.z, units = a.H + (a.v_from_k ? 1 : 2) * a.G;
  const int n = a.q_len[seq], i0 = blockIdx.y * HS_TILE, i1 = min(n, i0 + HS_TILE), slot = a.state_slot[seq];
  if (i0 >= n) return;
  if (slot < 0 || slot >= a.n_state) { if (threadIdx.x == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6E1); return; }
  float* x = xch[HALF ? warp : 0];
  if constexpr (!WHOLE) {
    const int unit = blockIdx.x * NWARP + warp;
    if (unit < units) conv_qkv_tile<T, V, TAPS, HALF, false>(a, unit, seq, i0, i1, slot, x, nullptr, nullptr);
  } else {
    __shared__ float part[2][NWARP][HS_TILE], inv[2][HS_TILE];
    for (int i = lane; i < 2 * HS_TILE; i += 32) part[i / HS_TILE][warp][i % HS_TILE] = 0.f;
    __syncwarp();
    for (int u = warp; u < a.H + a.G; u += NWARP) conv_qkv_tile<T, V, TAPS, HALF, true>(a, u, seq, i0, i1, slot, x, part[u < a.H ? 0 : 1][warp], nullptr);
    __syncthreads();
    if (threadIdx.x < 2 * HS_TILE) {
      const int which = threadIdx.x / HS_TILE, i = threadIdx.x % HS_TILE;
      float s = 0.f;
      for (int w = 0; w < NWARP; ++w) s += part[which][w][i];
      inv[which][i] = rsqrtf(s / (float)((which ? a.G : a.H) * a.dim) + a.eps);
    }
    __syncthreads();
    for (int u = warp; u < units; u += NWARP) conv_qkv_tile<T, V, TAPS, HALF, false>(a, u, seq, i0, i1, slot, x, nullptr, u < a.H + a.G ? inv[u < a.H ? 0 : 1] : nullptr);
  }
}

// ---------------------------------------------------------------- pooled blocks of long runs
// grid (blocks a run may complete, sequence): means of P cached rows, eight elements a thread.
template <typename T>
__global__ void __launch_bounds__(128) pool_kv_kernel(const T* __restrict__ cache, int row_stride, int n_slots, T* __restrict__ pooled, int pool_stride, int n_pooled, int width,
                                                      const AttnExtras<T> x, const int* __restrict__ page_table, int max_pages, const int* __restrict__ kv_len,
                                                      const int* __restrict__ q_len, int* status) {
  pdl_launch(); pdl_wait();
  const int seq = blockIdx.y, P = x.pool, kv = kv_len[seq], n = q_len[seq], b = (kv - n) / P + blockIdx.x;
  if (n <= HS_TILE || (long long)(b + 1) * P > kv) return;                // (short runs have left theirs)
  const int* table = page_table + (size_t)seq * max_pages;
  const int row_b = x.strip_row(b >> 3, table) + (b & 7);
  if (row_b < 0 || row_b >= n_pooled) { if (threadIdx.x == 0) ca_dev_fail(status, CA_DEV_BAD_INDEX, b & 0xFFFF); return; }
  for (int i = threadIdx.x * 8; i < width; i += 1024) {
    float m[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int p0 = b * P; p0 < (b + 1) * P; p0 += 4) {
      float u[4][8];
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int p = min(p0 + q, (b + 1) * P - 1), cs = min(max(table[p / 64] * 64 + p % 64, 0), n_slots - 1);
        load8<T>(cache + (size_t)cs * row_stride + i, u[q]);
      }
#pragma unroll
      for (int q = 0; q < 4; ++q)
        if (p0 + q < (b + 1) * P)
#pragma unroll
          for (int k = 0; k < 8; ++k) m[k] += u[q][k];
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) m[k] /= (float)P;
    store8<T>(pooled + (size_t)row_b * pool_stride + i, m);
  }
}

// ---------------------------------------------------------------- short convolution in front of the recurrence
template <typename T>
struct RecConv {
  const T* proj; int ldp;                       // rows whose columns [0, C) are the x branch
  const float* x_b; const float* w; const float* w_b;       // [C], [taps, C], [C]
  T* ring;                                      // [slots, R, C] projected rows (without x_b) by position
  const int* state_slot; const int* q_start; const int* q_len; const int* kv_len;
  T* u; int ldt, sq, sqp;                       // block-major operand: channel b * sq + j of row t at ((b * ldt) + t) * sqp + j
  int4* tiles; int* n_tiles;                    // tile table of the gate product: {block, first operand row, rows, 0}
  int T_rows, tn, C, taps, R, n_state;
  int* status;
};

template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(128) rglru_conv_kernel(const RecConv<T> a) {
  pdl_launch(); pdl_wait();
  if (blockIdx.x == 0 && blockIdx.y == 0 && blockIdx.z == 0 && a.tiles) {
    const int per = (a.T_rows + a.tn - 1) / a.tn, nt = a.C / a.sq * per;
    for (int i = threadIdx.x; i < nt; i += blockDim.x) {
      const int b = i / per, r0 = (i % per) * a.tn;
      a.tiles[i] = make_int4(b, b * a.ldt + r0, min(a.tn, a.T_rows - r0), 0);
    }
    if (threadIdx.x == 0) *a.n_tiles = nt;
  }
  const int ch = (blockIdx.x * blockDim.x + threadIdx.x) * V, seq = blockIdx.z;
  const int n = a.q_len[seq], i0 = blockIdx.y * HS_TILE;
  if (ch >= a.C || i0 >= n) return;
  const int row0 = a.q_start[seq], p0 = a.kv_len[seq] - n, slot = a.state_slot[seq], i1 = min(n, i0 + HS_TILE);
  if (slot < 0 || slot >= a.n_state) { if (ch == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6E2); return; }
  const int taps = TAPS ? TAPS : a.taps;
  T* ring = a.ring + (size_t)slot * a.R * a.C + ch;
  T* u = a.u + ((size_t)(ch / a.sq) * a.ldt + row0) * a.sqp + ch % a.sq;
  float xb[V], wb[V];
  load_v<float, V>(a.x_b + ch, xb); load_v<float, V>(a.w_b + ch, wb);
  auto raw = [&](int i, float* v) { load_v<T, V>(a.proj + (size_t)(row0 + i) * a.ldp + ch, v); };
  auto input = [&](int i, float* v) {
    const int pos = p0 + i;
    if (pos < 0) {
#pragma unroll
      for (int k = 0; k < V; ++k) v[k] = 0.f;
      return;
    }
    if (i >= 0) raw(i, v);
    else load_v<T, V>(ring + (size_t)(pos % a.R) * a.C, v);
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] += xb[k];
  };
  constexpr int NH = TAPS > 1 ? TAPS - 1 : 1, NW = TAPS ? TAPS : 1;
  float hist[NH][V], wr[NW][V];
  if (TAPS) {
#pragma unroll
    for (int j = 0; j < NW; ++j) load_v<float, V>(a.w + (size_t)j * a.C + ch, wr[j]);
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) input(i0 - (TAPS - 1) + j, hist[j]);
  }
  const bool keep = n <= a.R - (taps - 1);
  constexpr int NB = 4;                                 // rows loaded together
  for (int ib = i0; ib < i1; ib += NB) {
   float rows[NB][V];
#pragma unroll
   for (int q = 0; q < NB; ++q) raw(min(ib + q, i1 - 1), rows[q]);
#pragma unroll
   for (int q = 0; q < NB; ++q) {
    const int i = ib + q;
    if (i >= i1) break;
    float cur[V], y[V];
    const float* r = rows[q];
    if (keep) store_v<T, V>(ring + (size_t)((p0 + i) % a.R) * a.C, r);
#pragma unroll
    for (int k = 0; k < V; ++k) { cur[k] = r[k] + xb[k]; y[k] = wb[k]; }
    if (TAPS) {
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] = fmaf(wr[j][k], hist[j][k], y[k]);
#pragma unroll
      for (int k = 0; k < V; ++k) y[k] = fmaf(wr[NW - 1][k], cur[k], y[k]);
#pragma unroll
      for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
        for (int k = 0; k < V; ++k) hist[j][k] = hist[j + 1][k];
      if (TAPS > 1)
#pragma unroll
        for (int k = 0; k < V; ++k) hist[NH - 1][k] = cur[k];
    } else {
      for (int j = 0; j < taps; ++j) {
        float w[V], s[V];
        load_v<float, V>(a.w + (size_t)j * a.C + ch, w);
        input(i - (taps - 1) + j, s);
#pragma unroll
        for (int k = 0; k < V; ++k) y[k] = fmaf(w[k], s[k], y[k]);
      }
    }
    store_v<T, V>(u + (size_t)i * a.sqp, y);
   }
  }
  if (!keep && i0 == 0)
    for (int i = max(0, n - (taps - 1)); i < n; ++i) {
      float r[V];
      raw(i, r);
      store_v<T, V>(ring + (size_t)((p0 + i) % a.R) * a.C, r);
    }
}

// ---------------------------------------------------------------- real-gated linear recurrence
//   log a = decay * sigmoid(zr),  S <- a S + sqrt(1 - a^2) sigmoid(zi) u,  out = S * gelu(y)
template <typename T>
struct LruScan {
  const T* u; int ldt, sq, sqp;                 // block-major operand of the gate product
  float* gates; int ldg;                        // [T, ldg]: block b's decay gate at columns [2 b sq, + sq), input gate at the next sq; the
                                                // aggregate pass leaves {a - 1, input of the recurrence} in their places
  const float* gates_b; const float* decay;     // the same order; [C]
  const T* y; int ldy; const float* y_b;        // y branch rows and bias
  float* state;                                 // [slots, depth + 1, C] states by position
  const int* state_slot; const int* q_start; const int* q_len; const int* kv_len;
  float2* agg;                                  // chunk aggregates [.., C]: first chunk {state in front, state behind}, later ones {decay, sum}
  T* out; int ldo;
  int C, depth, n_state;
  int* status;
};

// fp32 results either way; beside bf16 operands the hardware's approximations (a few units in the last place) do.
template <typename T> __device__ __forceinline__ float sigmoid_t(float z);
template <> __device__ __forceinline__ float sigmoid_t<float>(float z) { return 1.f / (1.f + expf(-z)); }
template <> __device__ __forceinline__ float sigmoid_t<bf16>(float z) { return __fdividef(1.f, 1.f + __expf(-fmaxf(z, -80.f))); }
// two at the price of one reciprocal
template <typename T> __device__ __forceinline__ void sigmoid2_t(float x, float y, float& sx, float& sy);
template <> __device__ __forceinline__ void sigmoid2_t<float>(float x, float y, float& sx, float& sy) { sx = sigmoid_t<float>(x); sy = sigmoid_t<float>(y); }
template <> __device__ __forceinline__ void sigmoid2_t<bf16>(float x, float y, float& sx, float& sy) {
  const float ex = 1.f + __expf(-fmaxf(x, -40.f)), ey = 1.f + __expf(-fmaxf(y, -40.f)), inv = __fdividef(1.f, ex * ey);
  sx = inv * ey; sy = inv * ex;
}
// e^z - 1 for z <= 0: near zero the Taylor series (seven terms: relative error below 1e-7 down to z = -1/4), elsewhere the difference
template <typename T> __device__ __forceinline__ float expm1_t(float z);
template <> __device__ __forceinline__ float expm1_t<float>(float z) { return expm1f(z); }
template <> __device__ __forceinline__ float expm1_t<bf16>(float z) {
  float p = fmaf(z, 1.f / 7.f, 1.f);
  p = fmaf(z * (1.f / 6.f), p, 1.f); p = fmaf(z * 0.2f, p, 1.f); p = fmaf(z * 0.25f, p, 1.f); p = fmaf(z * (1.f / 3.f), p, 1.f); p = fmaf(z * 0.5f, p, 1.f);
  return z > -0.25f ? z * p : __expf(z) - 1.f;
}
template <typename T> __device__ __forceinline__ float sqrt_t(float z);
template <> __device__ __forceinline__ float sqrt_t<float>(float z) { return sqrtf(z); }
template <> __device__ __forceinline__ float sqrt_t<bf16>(float z) { return z * rsqrtf(fmaxf(z, 1e-30f)); }

// PASS 0: aggregates of every chunk but a run's last one; 1: outputs and states.
template <typename T, int V, int PASS>
__global__ void __launch_bounds__(128) lru_scan_kernel(const LruScan<T> a) {
  pdl_launch(); pdl_wait();
  constexpr int NB = 4;                         // rows loaded together: nothing but the state depends on the row before
  const int ch = (blockIdx.x * blockDim.x + threadIdx.x) * V, c = blockIdx.y, seq = blockIdx.z;
  const int n = a.q_len[seq], chunks = (n + HS_CHUNK - 1) / HS_CHUNK;
  if (ch >= a.C || c >= chunks || (PASS == 0 && c == chunks - 1)) return;
  const int row0 = a.q_start[seq], p0 = a.kv_len[seq] - n, slot = a.state_slot[seq];
  if (slot < 0 || slot >= a.n_state) { if (ch == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6E3); return; }
  const int b = ch / a.sq, j0 = ch % a.sq, gc = 2 * b * a.sq + j0;
  const T* u = a.u + ((size_t)b * a.ldt + row0) * a.sqp + j0;
  float* g = a.gates + (size_t)row0 * a.ldg + gc;
  float* st = a.state + (size_t)slot * (a.depth + 1) * a.C + ch;
  // aggregates of a run's chunks are consecutive rows; q_start / CHUNK + seq keeps the runs of a step apart
  float2* agg = a.agg + (size_t)(row0 / HS_CHUNK + seq) * a.C + ch;
  float rb[V], ib[V], dk[V], yb[V], h[V], A[V], h0[V];
  load_v<float, V>(a.gates_b + gc, rb); load_v<float, V>(a.gates_b + gc + a.sq, ib); load_v<float, V>(a.decay + ch, dk);
  if (PASS == 1) load_v<float, V>(a.y_b + ch, yb);
#pragma unroll
  for (int k = 0; k < V; ++k) { h[k] = 0.f; A[k] = 1.f; }
  if (c == 0 && (PASS == 0 || chunks == 1)) {
    if (p0 > 0) load_v<float, V>(st + (size_t)((p0 - 1) % (a.depth + 1)) * a.C, h);
  } else if (PASS == 1) {
    // the first chunk's entry holds both its ends, so no block reads the ring that the last chunk's block writes
#pragma unroll
    for (int k = 0; k < V; ++k) { const float2 f = agg[k]; h[k] = c == 0 ? f.x : f.y; }
    for (int q0 = 1; q0 < c; q0 += 8) {
      float2 f[8][V];
#pragma unroll
      for (int q = 0; q < 8; ++q)
#pragma unroll
        for (int k = 0; k < V; ++k) f[q][k] = q0 + q < c ? agg[(size_t)(q0 + q) * a.C + k] : make_float2(1.f, 0.f);
#pragma unroll
      for (int q = 0; q < 8; ++q)
#pragma unroll
        for (int k = 0; k < V; ++k) h[k] = fmaf(f[q][k].x, h[k], f[q][k].y);
    }
  }
#pragma unroll
  for (int k = 0; k < V; ++k) h0[k] = h[k];
  const int i1 = min(n, (c + 1) * HS_CHUNK);
  const bool ready = PASS == 1 && c < chunks - 1;       // the aggregate pass has been here
  for (int i0 = c * HS_CHUNK; i0 < i1; i0 += NB) {
    float zr[NB][V], zi[NB][V], us[NB][V], ys[NB][V];
#pragma unroll
    for (int q = 0; q < NB; ++q) {
      const int i = min(i0 + q, i1 - 1);
      load_v<float, V>(g + (size_t)i * a.ldg, zr[q]); load_v<float, V>(g + (size_t)i * a.ldg + a.sq, zi[q]);
      if (!ready) load_v<T, V>(u + (size_t)i * a.sqp, us[q]);
      if (PASS == 1) load_v<T, V>(a.y + (size_t)(row0 + i) * a.ldy + ch, ys[q]);
    }
#pragma unroll
    for (int q = 0; q < NB; ++q) {
      const int i = i0 + q;
      if (i >= i1) break;
      float o[V], m[V], in[V];
      if (ready) {
#pragma unroll
        for (int k = 0; k < V; ++k) { m[k] = zr[q][k]; in[k] = zi[q][k]; }
      } else {
#pragma unroll
        for (int k = 0; k < V; ++k) {
          float la, gate;
          sigmoid2_t<T>(zr[q][k] + rb[k], zi[q][k] + ib[k], la, gate);
          // with m = a - 1: a S = S + m S and 1 - a^2 = -m (m + 2), both exact to rounding where a is close to 1 (long memories)
          m[k] = expm1_t<T>(la * dk[k]);
          in[k] = sqrt_t<T>(-m[k] * (m[k] + 2.f)) * gate * us[q][k];
        }
      }
      if (PASS == 0) { store_v<float, V>(g + (size_t)i * a.ldg, m); store_v<float, V>(g + (size_t)i * a.ldg + a.sq, in); }
#pragma unroll
      for (int k = 0; k < V; ++k) {
        h[k] = fmaf(m[k], h[k], h[k]) + in[k];
        if (PASS == 0) A[k] = fmaf(m[k], A[k], A[k]);
        if (PASS == 1) {
          const float z = ys[q][k] + yb[k];
          o[k] = h[k] * z * sigmoid_t<T>(1.5957691216057308f * fmaf(0.044715f * z * z, z, z));      // 0.5 (1 + tanh(w)) = sigmoid(2 w)
        }
      }
      if (PASS == 1) {
        store_v<T, V>(a.out + (size_t)(row0 + i) * a.ldo + ch, o);
        if (n <= a.depth || i == n - 1) store_v<float, V>(st + (size_t)((p0 + i) % (a.depth + 1)) * a.C, h);
      }
    }
  }
  if (PASS == 0)
#pragma unroll
    for (int k = 0; k < V; ++k) agg[(size_t)c * a.C + k] = make_float2(c == 0 ? h0[k] : A[k], h[k]);
}

// ---------------------------------------------------------------- clamped GLU over two projected rows
template <typename T>
__global__ void glu_rows_kernel(const T* __restrict__ g, const T* __restrict__ u, const float* __restrict__ gb, const float* __restrict__ ub, T* __restrict__ out,
                                int ldi, int ldo, int N, float limit) {
  pdl_launch(); pdl_wait();
  const int t = blockIdx.x;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < N; i += gridDim.y * blockDim.x) {
    const float gv = fminf(to_f(g[(size_t)t * ldi + i]) + gb[i], limit), uv = fminf(fmaxf(to_f(u[(size_t)t * ldi + i]) + ub[i], -limit), limit);
    out[(size_t)t * ldo + i] = to_t<T>(gv / (1.f + expf(-1.702f * gv)) * (uv + 1.f));
  }
}

// ---------------------------------------------------------------- windowed grouped-query attention on the ordinary cores
// One block per (query row, head): scores of a page of keys (a warp takes 16 of them), online softmax, weighted sum of the page's values
// (a thread owns columns tid, tid + 128, ...).
#define WA_COLS 4
template <typename T>
__global__ void __launch_bounds__(128) window_attn_simt_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ cache, const int* __restrict__ page_table,
                                                               const int* __restrict__ kv_len, const int* __restrict__ q_start, const int* __restrict__ q_len,
                                                               T* __restrict__ out, int ldo, int n_seq, int G, int group, int dp, int dvp, int dv, int row_stride, int pool_stride,
                                                               int max_pages, int n_slots, int window, float scale, const AttnExtras<T> x, int* status) {
  pdl_launch(); pdl_wait();
  extern __shared__ float qs[];
  __shared__ float sc[64];
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, kh = h / group;
  int seq = -1;
  for (int s = 0; s < n_seq; ++s) if (t >= q_start[s] && t < q_start[s] + q_len[s]) { seq = s; break; }
  if (seq < 0) return;
  const int pos = kv_len[seq] - q_len[seq] + t - q_start[seq], lo = window > 0 ? max(0, pos - window + 1) : 0;
  const T* qr = q + (size_t)t * q_stride + (size_t)h * dp;
  for (int i = tid; i < dp; i += 128) qs[i] = to_f(qr[i]);
  __syncthreads();
  float m = -INFINITY, l = 0.f, o[WA_COLS];
#pragma unroll
  for (int j = 0; j < WA_COLS; ++j) o[j] = 0.f;
  // pages of kept first keys that lie in front of the window, or tiles of pooled blocks, then the window's
  const int kept = x.lead_tiles(lo / 64, 64, pos, window), pages = kept + pos / 64 - lo / 64 + 1, blocks = x.blocks_seen(pos, window);
  __shared__ int strip[8];
  for (int pi = 0; pi < pages; ++pi) {
    const bool pooled = x.pool > 0 && pi < kept;
    const int k0 = (pi < kept ? pi : pi - kept + lo / 64) * 64;
    int slot0 = 0;
    if (pooled) {
      if (tid < 8) strip[tid] = x.strip_row(min(k0 / 8 + tid, (blocks - 1) >> 3), page_table + (size_t)seq * max_pages);
      __syncthreads();
    } else {
      slot0 = page_table[(size_t)seq * max_pages + k0 / 64] * 64;
      if (slot0 < 0 || slot0 + 64 > n_slots) { if (tid == 0) ca_dev_fail(status, CA_DEV_BAD_INDEX, t); slot0 = 0; }
    }
    auto row_of = [&](int j) -> const T* {
      return pooled ? x.pooled + (size_t)(strip[j >> 3] + (j & 7)) * pool_stride : cache + (size_t)(slot0 + j) * row_stride;
    };
    const int n = min(64, pooled ? blocks - k0 : pos + 1 - k0);
    for (int j = warp * 16; j < warp * 16 + 16; ++j) {
      float s = 0.f;
      const bool in = j < n && (pooled || k0 + j >= lo || k0 + j < x.keep_first);
      if (in) {
        const T* kb = row_of(j) + (size_t)kh * dp;
        for (int i = lane; i < dp; i += 32) s = fmaf(qs[i], to_f(kb[i]), s);
      }
      s = warp_sum(s);
      if (lane == 0) sc[j] = in ? s * scale : -INFINITY;
    }
    __syncthreads();
    const float s0 = sc[lane], s1 = sc[lane + 32];
    const float mn = fmaxf(m, warp_max(fmaxf(s0, s1)));             // every page of the loop holds a visible key, so mn is finite
    const float al = m == -INFINITY ? 0.f : expf(m - mn);
    const float e0 = expf(s0 - mn), e1 = expf(s1 - mn);
    l = l * al + warp_sum(e0 + e1);
    m = mn;
    __syncthreads();
    if (warp == 0) { sc[lane] = e0; sc[lane + 32] = e1; }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < WA_COLS; ++c) {
      const int i = tid + c * 128;
      if (i < dv) {
        float acc = o[c] * al;
        for (int j = 0; j < n; ++j) acc = fmaf(sc[j], to_f(row_of(j)[(size_t)G * dp + (size_t)kh * dvp + i]), acc);         // keys out of sight weigh zero
        o[c] = acc;
      }
    }
    __syncthreads();
  }
  if (x.sink) l += expf(x.sink[h] - m);
  const float f = (l > 0.f ? 1.f / l : 0.f) * x.head_factor(t, h);
#pragma unroll
  for (int c = 0; c < WA_COLS; ++c) {
    const int i = tid + c * 128;
    if (i < dv) out[(size_t)t * ldo + (size_t)h * dv + i] = to_t<T>(o[c] * f * x.value_factor(t, h * dv + i));
  }
}

// ---------------------------------------------------------------- C ABI
struct CaNormRows {
  float* x; const int* tokens; const void* table; const void* add; const float* bias; const float* post; const int* src_rows; const float* gain; void* xn; int* status;
  int W, Wp, vocab, ldn, raw; float mult, eps, scale;
};

template <typename T, int MODE>
static int norm_rows_launch(const CaNormRows* c, int rows, cudaStream_t s) {
  const NormRows<T> a{c->x, c->W, c->Wp, c->tokens, (const bf16*)c->table, c->vocab, c->scale, (const T*)c->add, c->bias, c->post, c->mult, c->src_rows, c->gain, (T*)c->xn, c->ldn, c->raw, c->eps, c->status};
  const int chunks = c->Wp / 8, most = rows <= 2 * ca_sm_count() ? 1024 : 256;
  int nt = chunks <= most ? (chunks + 31) / 32 * 32 : most;
  if ((chunks + nt - 1) / nt > 8) nt = 1024;
  const int nch = (chunks + nt - 1) / nt;
  if (nch == 1) CA_LAUNCH_PDL((norm_rows_kernel<T, 1, MODE>), rows, nt, 0, s, a);
  else if (nch == 2) CA_LAUNCH_PDL((norm_rows_kernel<T, 2, MODE>), rows, nt, 0, s, a);
  else if (nch <= 4) CA_LAUNCH_PDL((norm_rows_kernel<T, 4, MODE>), rows, nt, 0, s, a);
  else if (nch <= 8) CA_LAUNCH_PDL((norm_rows_kernel<T, 8, MODE>), rows, nt, 0, s, a);
  else return ca_fail(CA_ERR_ARG, "norm_rows: rows of %d elements (at most 65536)", c->Wp);
  CA_CHECK_LAUNCH("norm_rows");
  return CA_OK;
}

extern "C" int cuteafd_norm_rows(const CaNormRows* c, int mode, int rows, int f32, cudaStream_t s) {
  CA_REQUIRE(c && c->x && c->W >= 1 && c->Wp >= c->W && c->Wp % 8 == 0 && (!c->xn || (c->ldn % 8 == 0 && c->ldn >= c->Wp)), "norm_rows: bad arguments");
  CA_REQUIRE(mode == ROWS_EMBED ? c->tokens && c->table && c->vocab > 0 : mode == ROWS_ADD ? c->add && (!c->table || (c->tokens && c->vocab > 0)) : mode == ROWS_GATHER && c->src_rows && c->xn, "norm_rows: mode %d without its inputs", mode);
  if (rows <= 0) return CA_OK;
  if (mode == ROWS_EMBED) return f32 ? norm_rows_launch<float, ROWS_EMBED>(c, rows, s) : norm_rows_launch<bf16, ROWS_EMBED>(c, rows, s);
  if (mode == ROWS_ADD) return f32 ? norm_rows_launch<float, ROWS_ADD>(c, rows, s) : norm_rows_launch<bf16, ROWS_ADD>(c, rows, s);
  return f32 ? norm_rows_launch<float, ROWS_GATHER>(c, rows, s) : norm_rows_launch<bf16, ROWS_GATHER>(c, rows, s);
}

extern "C" int cuteafd_rope_table(const int* positions, const float* freq, float amp, int pairs, void* out, int T, cudaStream_t s) {
  CA_REQUIRE(positions && freq && out && pairs >= 1, "rope_table: bad arguments");
  if (T <= 0) return CA_OK;
  CA_LAUNCH_PDL(rope_table_kernel, T, pairs < 128 ? (pairs + 31) / 32 * 32 : 128, 0, s, positions, freq, amp, pairs, (float2*)out);
  CA_CHECK_LAUNCH("rope_table");
  return CA_OK;
}

struct CaConvQkv {
  const void* proj; const float* w; const float* bias; const float* q_norm; const float* k_norm; const void* rope; void* ring; const int* state_slot; const int* q_start;
  const int* q_len; const int* kv_len; const int* slot_map; void* q; void* cache; int* status; void* pooled; const int* page_table;
  int ldp, q_stride, row_stride, n_slots, H, G, dim, dp, vdim, dvp, pairs, taps, R, C, n_state, n_seq, max_q_len, norm, half, v_from_k, pool, pool_rows, pool_stride, n_pooled, max_pages; float eps;
};

template <typename T>
static AttnExtras<T> pool_extras(int pool, int pool_rows) {
  AttnExtras<T> x = attn_extras<T>(nullptr, 0);
  x.pool = pool; x.pool_rows = pool_rows;
  return x;
}

template <typename T, int V, bool HALF, bool WHOLE>
static int conv_qkv_launch(const CaConvQkv* c, cudaStream_t s) {
  const ConvQkv<T> a{(const T*)c->proj, c->ldp, c->w, c->bias, c->q_norm, c->k_norm, (const float2*)c->rope, (T*)c->ring, c->state_slot, c->q_start, c->q_len, c->kv_len,
                     c->slot_map, (T*)c->q, c->q_stride, (T*)c->cache, c->row_stride, c->n_slots, c->H, c->G, c->dim, c->dp, c->vdim, c->dvp, c->pairs, c->taps, c->R, c->C,
                     c->n_state, c->norm, c->v_from_k, c->eps, c->status, pool_extras<T>(c->pool, c->pool_rows), (T*)c->pooled, c->page_table, c->max_pages, c->pool_stride, c->n_pooled};
  const int units = c->H + (c->v_from_k ? 1 : 2) * c->G;
  const dim3 grid(WHOLE ? 1 : (units + 3) / 4, (c->max_q_len + HS_TILE - 1) / HS_TILE, c->n_seq);
  const int nt = WHOLE ? HS_WHOLE_WARPS * 32 : 128;
  if (c->taps == 1) CA_LAUNCH_PDL((conv_qkv_kernel<T, V, 1, HALF, WHOLE>), grid, nt, 0, s, a);
  else if (c->taps == 2) CA_LAUNCH_PDL((conv_qkv_kernel<T, V, 2, HALF, WHOLE>), grid, nt, 0, s, a);
  else if (c->taps == 3) CA_LAUNCH_PDL((conv_qkv_kernel<T, V, 3, HALF, WHOLE>), grid, nt, 0, s, a);
  else if (c->taps == 4) CA_LAUNCH_PDL((conv_qkv_kernel<T, V, 4, HALF, WHOLE>), grid, nt, 0, s, a);
  else CA_LAUNCH_PDL((conv_qkv_kernel<T, V, 0, HALF, WHOLE>), grid, nt, 0, s, a);
  CA_CHECK_LAUNCH("conv_qkv");
  return CA_OK;
}

template <typename T, int V>
static int conv_qkv_modes(const CaConvQkv* c, cudaStream_t s) {
  if (c->norm == QK_NORM_WHOLE) return c->half ? conv_qkv_launch<T, V, true, true>(c, s) : conv_qkv_launch<T, V, false, true>(c, s);
  return c->half ? conv_qkv_launch<T, V, true, false>(c, s) : conv_qkv_launch<T, V, false, false>(c, s);
}

extern "C" int cuteafd_conv_qkv(const CaConvQkv* c, int f32, cudaStream_t s) {
  CA_REQUIRE(c && c->proj && c->state_slot && c->q_start && c->q_len && c->kv_len && c->slot_map && c->q, "conv_qkv: null argument");
  CA_REQUIRE(c->taps >= 1 && c->taps <= HS_MAX_TAPS && (c->taps == 1 || (c->w && c->ring)) && (!c->ring || c->R >= c->taps), "conv_qkv: convolution without its weights or inputs");
  CA_REQUIRE(c->norm >= QK_NORM_NONE && c->norm <= QK_NORM_WHOLE && (c->norm != QK_NORM_WHOLE || (c->q_norm && (c->G == 0 || c->k_norm))) && (c->G == 0 || !c->q_norm == !c->k_norm), "conv_qkv: norm without its gains");
  CA_REQUIRE(!c->pooled || (c->pool >= 1 && c->pool_rows == (8 + c->pool - 1) / c->pool * 8 && c->page_table && !c->v_from_k && c->G >= 1 && c->pool_stride >= c->G * (c->dp + c->dvp) && c->pool_stride % 8 == 0),
             "conv_qkv: pooled blocks without their rows and pages");
  CA_REQUIRE(c->H >= 1 && c->G >= 0 && (c->G == 0 || c->cache) && (!c->v_from_k || c->vdim == c->dim), "conv_qkv: bad geometry");
  CA_REQUIRE(c->dim >= 1 && c->dim <= 256 && c->vdim <= 256 && c->dp % 8 == 0 && c->dvp % 8 == 0 && c->dim <= c->dp && c->vdim <= c->dvp && c->row_stride % 8 == 0, "conv_qkv: heads of up to 256 dimensions");
  CA_REQUIRE(c->C == (c->H + c->G) * c->dim + (c->v_from_k ? 0 : c->G * c->vdim) && c->ldp >= c->C && c->q_stride >= c->H * c->dp && (c->G == 0 || c->row_stride >= c->G * (c->dp + c->dvp)), "conv_qkv: row too short");
  CA_REQUIRE(c->pairs >= 0 && 2 * c->pairs <= c->dim && (c->pairs == 0 || c->rope) && (!c->ring || c->R - (c->taps - 1) <= HS_TILE), "conv_qkv: bad rotation or ring");
  if (c->n_seq <= 0 || c->max_q_len <= 0) return CA_OK;
  CA_REQUIRE(c->n_seq <= 65535 && (c->max_q_len + HS_TILE - 1) / HS_TILE <= 65535, "conv_qkv: step too large");
  const int nc = ((c->dim > c->vdim || c->G == 0 ? c->dim : c->vdim) + 63) / 64;
  if (nc <= 1) return f32 ? conv_qkv_modes<float, 2>(c, s) : conv_qkv_modes<bf16, 2>(c, s);
  if (nc <= 2) return f32 ? conv_qkv_modes<float, 4>(c, s) : conv_qkv_modes<bf16, 4>(c, s);
  return f32 ? conv_qkv_modes<float, 8>(c, s) : conv_qkv_modes<bf16, 8>(c, s);
}

// Blocks that runs of more than HS_TILE tokens complete (shorter runs: `cuteafd_conv_qkv` leaves them).
extern "C" int cuteafd_pool_kv(const void* cache, int row_stride, int n_slots, void* pooled, int pool_stride, int n_pooled, int width, int pool, int pool_rows, const int* page_table,
                               int max_pages, const int* kv_len, const int* q_len, int n_seq, int max_q_len, int f32, int* status, cudaStream_t s) {
  CA_REQUIRE(cache && pooled && page_table && kv_len && q_len && pool >= 1 && pool_rows == (8 + pool - 1) / pool * 8, "pool_kv: bad arguments");
  CA_REQUIRE(width % 8 == 0 && width <= row_stride && width <= pool_stride && row_stride % 8 == 0 && pool_stride % 8 == 0 && n_slots >= 1, "pool_kv: rows too short");
  if (n_seq <= 0 || max_q_len <= HS_TILE) return CA_OK;
  CA_REQUIRE(n_seq <= 65535, "pool_kv: too many sequences");
  const dim3 grid(max_q_len / pool + 1, n_seq);
  if (f32) CA_LAUNCH_PDL(pool_kv_kernel<float>, grid, 128, 0, s, (const float*)cache, row_stride, n_slots, (float*)pooled, pool_stride, n_pooled, width, pool_extras<float>(pool, pool_rows), page_table, max_pages, kv_len, q_len, status);
  else CA_LAUNCH_PDL(pool_kv_kernel<bf16>, grid, 128, 0, s, (const bf16*)cache, row_stride, n_slots, (bf16*)pooled, pool_stride, n_pooled, width, pool_extras<bf16>(pool, pool_rows), page_table, max_pages, kv_len, q_len, status);
  CA_CHECK_LAUNCH("pool_kv");
  return CA_OK;
}

struct CaRecurrence {          // one recurrent layer's step: shared by its convolution and its scan
  const void* x; const void* y; const float* x_b; const float* y_b; const float* conv; const float* conv_b; void* ring; float* state; void* u; float* gates;
  const float* gates_b; const float* decay; void* agg; void* out; void* tiles; int* n_tiles; const int* state_slot; const int* q_start; const int* q_len; const int* kv_len;
  int* status;
  int ldp, ldt, sq, sqp, ldg, ldo, tn, T, C, taps, depth, n_state, n_seq, max_q_len, agg_rows;
};

template <typename T, int V>
static int rglru_conv_launch(const CaRecurrence* c, cudaStream_t s) {
  const RecConv<T> a{(const T*)c->x, c->ldp, c->x_b, c->conv, c->conv_b, (T*)c->ring, c->state_slot, c->q_start, c->q_len, c->kv_len, (T*)c->u, c->ldt, c->sq, c->sqp,
                     (int4*)c->tiles, c->n_tiles, c->T, c->tn, c->C, c->taps, c->taps - 1 + c->depth, c->n_state, c->status};
  const dim3 grid((c->C / V + 127) / 128, (c->max_q_len + HS_TILE - 1) / HS_TILE, c->n_seq);
  if (c->taps == 2) CA_LAUNCH_PDL((rglru_conv_kernel<T, V, 2>), grid, 128, 0, s, a);
  else if (c->taps == 3) CA_LAUNCH_PDL((rglru_conv_kernel<T, V, 3>), grid, 128, 0, s, a);
  else if (c->taps == 4) CA_LAUNCH_PDL((rglru_conv_kernel<T, V, 4>), grid, 128, 0, s, a);
  else CA_LAUNCH_PDL((rglru_conv_kernel<T, V, 0>), grid, 128, 0, s, a);
  CA_CHECK_LAUNCH("rglru_conv");
  return CA_OK;
}

template <typename T, int V>
static int lru_scan_launch(const CaRecurrence* c, cudaStream_t s) {
  const LruScan<T> a{(const T*)c->u, c->ldt, c->sq, c->sqp, c->gates, c->ldg, c->gates_b, c->decay, (const T*)c->y, c->ldp, c->y_b, c->state, c->state_slot, c->q_start,
                     c->q_len, c->kv_len, (float2*)c->agg, (T*)c->out, c->ldo, c->C, c->depth, c->n_state, c->status};
  const int chunks = (c->max_q_len + HS_CHUNK - 1) / HS_CHUNK;
  const dim3 grid((c->C / V + 127) / 128, chunks, c->n_seq);
  if (chunks > 1) {
    CA_LAUNCH_PDL((lru_scan_kernel<T, V, 0>), dim3(grid.x, chunks - 1, c->n_seq), 128, 0, s, a);
    CA_CHECK_LAUNCH("lru_scan aggregates");
  }
  CA_LAUNCH_PDL((lru_scan_kernel<T, V, 1>), grid, 128, 0, s, a);
  CA_CHECK_LAUNCH("lru_scan");
  return CA_OK;
}

static bool recurrence_ok(const CaRecurrence* c) {
  return c && c->state_slot && c->q_start && c->q_len && c->kv_len && c->u && c->C >= 1 && c->sq >= 1 && c->C % c->sq == 0 && c->sqp >= c->sq && c->ldt >= c->T &&
         c->taps >= 1 && c->taps <= HS_MAX_TAPS && c->depth >= 1 && c->depth <= HS_TILE && c->n_state >= 1 && c->n_seq <= 65535 && c->max_q_len <= 65535 * HS_TILE;
}

extern "C" int cuteafd_rglru_conv(const CaRecurrence* c, int f32, cudaStream_t s) {
  CA_REQUIRE(recurrence_ok(c) && c->x && c->x_b && c->conv && c->conv_b && c->ring && (!c->tiles || (c->n_tiles && c->tn >= 1)) && c->ldp >= c->C, "rglru_conv: bad arguments");
  if (c->n_seq <= 0 || c->max_q_len <= 0) return CA_OK;
  const bool v4 = c->sq % 4 == 0 && c->sqp % 4 == 0 && c->ldp % 4 == 0 && ((uintptr_t)c->x & 15) == 0;
  if (v4) return f32 ? rglru_conv_launch<float, 4>(c, s) : rglru_conv_launch<bf16, 4>(c, s);
  return f32 ? rglru_conv_launch<float, 1>(c, s) : rglru_conv_launch<bf16, 1>(c, s);
}

extern "C" int cuteafd_lru_scan(const CaRecurrence* c, int f32, cudaStream_t s) {
  CA_REQUIRE(recurrence_ok(c) && c->gates && c->gates_b && c->decay && c->y && c->y_b && c->state && c->out && c->ldg >= 2 * c->C && c->ldo >= c->C && c->ldp >= c->C, "lru_scan: bad arguments");
  if (c->n_seq <= 0 || c->max_q_len <= 0) return CA_OK;
  CA_REQUIRE(c->max_q_len <= HS_CHUNK || (c->agg && c->agg_rows >= c->T / HS_CHUNK + c->n_seq + 1), "lru_scan: runs of more than %d tokens need room for their aggregates", HS_CHUNK);
  const bool v2 = c->sq % 2 == 0 && c->sqp % 2 == 0 && c->ldp % 2 == 0 && c->ldo % 2 == 0 && c->ldg % 2 == 0 && ((uintptr_t)c->y & 7) == 0;
  if (v2) return f32 ? lru_scan_launch<float, 2>(c, s) : lru_scan_launch<bf16, 2>(c, s);
  return f32 ? lru_scan_launch<float, 1>(c, s) : lru_scan_launch<bf16, 1>(c, s);
}

extern "C" int cuteafd_glu_rows(const void* g, const void* u, const float* gb, const float* ub, void* out, int T, int ldi, int ldo, int N, float limit, int f32, cudaStream_t s) {
  CA_REQUIRE(g && u && gb && ub && out && N >= 1 && ldi >= N && ldo >= N, "glu_rows: bad arguments");
  if (T <= 0) return CA_OK;
  const dim3 grid(T, (N + 1023) / 1024);
  if (f32) CA_LAUNCH_PDL(glu_rows_kernel<float>, grid, 256, 0, s, (const float*)g, (const float*)u, gb, ub, (float*)out, ldi, ldo, N, limit);
  else CA_LAUNCH_PDL(glu_rows_kernel<bf16>, grid, 256, 0, s, (const bf16*)g, (const bf16*)u, gb, ub, (bf16*)out, ldi, ldo, N, limit);
  CA_CHECK_LAUNCH("glu_rows");
  return CA_OK;
}

extern "C" int cuteafd_window_attention_simt(const void* q, int q_stride, const void* cache, const int* page_table, const int* kv_len, const int* q_start, const int* q_len,
                                             void* out, int ldo, int T, int n_seq, int Hq, int Hkv, int dp, int dvp, int dv, int row_stride, int pool_stride, int max_pages, int n_slots,
                                             int window, float scale, int f32, const CaAttnExtras* extras, int* status, cudaStream_t s) {
  CA_REQUIRE(q && cache && page_table && kv_len && q_start && q_len && out, "window_attention_simt: null argument");
  CA_REQUIRE(Hkv >= 1 && Hq % Hkv == 0 && Hq <= 65535 && dv >= 1 && dv <= dvp && dv <= 128 * WA_COLS && dp >= 1 && dp <= 4096 && row_stride >= Hkv * (dp + dvp) && ldo >= Hq * dv,
             "window_attention_simt: bad shape");
  CA_REQUIRE(attn_extras_ok(extras, false) && (!extras || !extras->pool || pool_stride >= Hkv * (dp + dvp)), "window_attention_simt: pooled blocks without their rows, or beside kept keys");
  if (T <= 0 || n_seq <= 0) return CA_OK;
  if (f32) CA_LAUNCH_PDL(window_attn_simt_kernel<float>, dim3(T, Hq), 128, dp * sizeof(float), s, (const float*)q, q_stride, (const float*)cache, page_table, kv_len, q_start, q_len, (float*)out, ldo, n_seq, Hkv, Hq / Hkv, dp, dvp, dv, row_stride, pool_stride, max_pages, n_slots, window, scale, attn_extras<float>(extras, window), status);
  else CA_LAUNCH_PDL(window_attn_simt_kernel<bf16>, dim3(T, Hq), 128, dp * sizeof(float), s, (const bf16*)q, q_stride, (const bf16*)cache, page_table, kv_len, q_start, q_len, (bf16*)out, ldo, n_seq, Hkv, Hq / Hkv, dp, dvp, dv, row_stride, pool_stride, max_pages, n_slots, window, scale, attn_extras<bf16>(extras, window), status);
  CA_CHECK_LAUNCH("window_attention_simt");
  return CA_OK;
}

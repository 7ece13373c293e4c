// Glue of the latent-attention layer stacks (parallel layers, fp32 residual rows, Dynamic Tanh in the place of a norm, looped layer
// ranges): everything between two matrix products is one launch, and every kernel that produces residual rows also writes the next
// product's operand - the normalised row, or the first half of the [x; x0] operand that opens a pass of the loop.
//   stack_embed      token row + position row -> residual (and the x0 half of the loop operand)
//   stack_stream     residual += a per-channel vector; or a gather of the rows that need logits
//   stack_combine    residual += ls1 * mixer output + ls2 * weighted sum of the routed experts' rows
//   latent_prepare   fused input projection (fp32: queries | latent | head gates | router logits) -> head-major queries, RMS-normed
//                    latent row in the paged cache, sigmoid gates, router logits, tile table of the per-head matrix products
//   latent_down      fused down-projections (fp32: queries' latent | latent, rotated key part) -> RMS-normed operand of the query expansion, cache row
//   latent_split     expanded queries -> head-major unrotated parts, rotated parts, tile table of the per-head products
//   latent_attn_simt absorbed attention for what the tcgen05 kernels do not take (fp32, ranks above 512, more than 128 heads)
// T is the type of the matrix-product operands and of the cache: bf16, or float for the all-fp32 mode.  Rows are padded to multiples of
// 8 elements (pad weights are zero).  (No counterpart in the reference, which has no such family; the fused shapes follow moe.cu.)
#include "stack_rows.cuh"

// What a row-producing kernel hands to the next matrix product: tanh(alpha x) w + b -> xn and / or the plain row -> cat.
template <typename T>
struct Emit {
  const float* w; const float* b; float alpha; T* xn; int ldn; T* cat; int ldc;
  __device__ __forceinline__ void operator()(const float* v, size_t row, int i) const {
    if (xn) {
      float nw[8], nb[8], y[8];
      load8<float>(w + i, nw); load8<float>(b + i, nb);
#pragma unroll
      for (int j = 0; j < 8; ++j) y[j] = fmaf(tanhf(alpha * v[j]), nw[j], nb[j]);
      store8<T>(xn + row * ldn + i, y);
    }
    if (cat) store8<T>(cat + row * ldc + i, v);
  }
};

template <typename T>
__global__ void stack_embed_kernel(const int* __restrict__ tokens, const int* __restrict__ positions, const bf16* __restrict__ table,
                                   const bf16* __restrict__ pos_table, float* __restrict__ x, T* __restrict__ x0, int ld0, int W, int vocab,
                                   int n_pos, int* status, const Emit<T> emit) {
  pdl_launch(); pdl_wait();
  const int t = blockIdx.x, i = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (i >= W) return;
  int tok = tokens[t], pos = positions[t];
  if (tok < 0 || tok >= vocab) { if (i == 0) ca_dev_fail(status, CA_DEV_BAD_INDEX, t); tok = 0; }
  float v[8], p[8];
  load8<bf16>(table + (size_t)tok * W + i, v);
  if (pos_table) {
    if (pos < 0 || pos >= n_pos) { if (i == 0) ca_dev_fail(status, CA_DEV_BAD_INDEX, t); pos = 0; }
    load8<bf16>(pos_table + (size_t)pos * W + i, p);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] += p[j];
  }
  store8<float>(x + (size_t)t * W + i, v);
  if (x0) store8<T>(x0 + (size_t)t * ld0 + i, v);
  emit(v, t, i);
}

template <typename T>
__global__ void stack_stream_kernel(float* __restrict__ x, const float* __restrict__ vec, const int* __restrict__ src_rows, int W, const Emit<T> emit) {
  pdl_launch(); pdl_wait();
  const int t = blockIdx.x, i = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (i >= W) return;
  const size_t row = src_rows ? (size_t)src_rows[t] : (size_t)t;
  float v[8];
  load8<float>(x + row * W + i, v);
  if (vec) {
    float a[8];
    load8<float>(vec + i, a);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] += a[j];
    store8<float>(x + row * W + i, v);
  }
  emit(v, t, i);
}

template <typename T>
__global__ void stack_combine_kernel(float* __restrict__ x, const T* __restrict__ mix, const float* __restrict__ ls1, const T* __restrict__ y,
                                     const int* __restrict__ slot_row, const float* __restrict__ wts, const float* __restrict__ ls2, int k, int W,
                                     const Emit<T> emit) {
  pdl_launch(); pdl_wait();
  const int t = blockIdx.x, i = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
  if (i >= W) return;
  float v[8], m[8], s[8], acc[8];
  load8<float>(x + (size_t)t * W + i, v);
  load8<T>(mix + (size_t)t * W + i, m);
  load8<float>(ls1 + i, s);
#pragma unroll
  for (int j = 0; j < 8; ++j) acc[j] = s[j] * m[j];
  if (k > 0) {
    float e[8], s2[8];
    load8<float>(ls2 + i, s2);
#pragma unroll
    for (int j = 0; j < 8; ++j) e[j] = 0.f;
    // eight routes at a time: row numbers and weights first, then all rows in flight together (as moe.cu::combine_routes8)
    for (int s0 = 0; s0 < k; s0 += 8) {
      int r[8]; float w[8], q[8][8];
#pragma unroll
      for (int j = 0; j < 8; ++j) { r[j] = (s0 + j < k) ? slot_row[(size_t)t * k + s0 + j] : -1; w[j] = (s0 + j < k) ? wts[(size_t)t * k + s0 + j] : 0.f; }
#pragma unroll
      for (int j = 0; j < 8; ++j) if (r[j] >= 0) load8<T>(y + (size_t)r[j] * W + i, q[j]);
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (r[j] >= 0) {
#pragma unroll
          for (int c = 0; c < 8; ++c) e[c] = fmaf(w[j], q[j][c], e[c]);
        }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j] = fmaf(s2[j], e[j], acc[j]);
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) v[j] += acc[j];
  store8<float>(x + (size_t)t * W + i, v);
  emit(v, t, i);
}

// ---------------------------------------------------------------- after the fused input projection
struct LatentPrep {
  const float* proj; int ldp;                    // [T, ldp] fp32: H * d queries | r latent | H gates (if any) | E router logits (if any)
  const float* norm_w; const int* slot_map;
  float* gate; float* logits;                    // [T, H] sigmoid, [T, E]
  int4* tiles; int* n_tiles;                     // tile table of the products grouped over heads: {head, first row, rows, 0}
  int* status;
  int T, ldt, H, d, dp, r, rp, row_stride, n_slots, E, tn, has_gate;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_prepare_kernel(const LatentPrep a, T* __restrict__ q, T* __restrict__ cache) {
  pdl_launch(); pdl_wait();
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  const float* row = a.proj + (size_t)t * a.ldp;
  const int slot = a.slot_map[t], Hd = a.H * a.d;
  const bool ok = slot >= 0 && slot < a.n_slots;
  if (!ok && tid == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, t);
  if (a.d % 4 == 0) {
    for (int i = tid * 4; i < Hd; i += nt * 4) {
      const float4 v = *(const float4*)(row + i);
      T o[4] = {to_t<T>(v.x), to_t<T>(v.y), to_t<T>(v.z), to_t<T>(v.w)};
      T* dst = q + ((size_t)(i / a.d) * a.ldt + t) * a.dp + i % a.d;
      if (sizeof(T) == 2) *(uint2*)dst = *(const uint2*)o; else *(uint4*)dst = *(const uint4*)o;
    }
  } else {
    for (int i = tid; i < Hd; i += nt) q[((size_t)(i / a.d) * a.ldt + t) * a.dp + i % a.d] = to_t<T>(row[i]);
  }
  const float* lat = row + Hd;
  float ss = 0.f;
  for (int i = tid; i < a.r; i += nt) ss += lat[i] * lat[i];
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.r + a.eps);
  if (ok) {
    T* dst = cache + (size_t)slot * a.row_stride;
    for (int i = tid; i < a.rp; i += nt) dst[i] = i < a.r ? to_t<T>(lat[i] * inv * a.norm_w[i]) : to_t<T>(0.f);
  }
  const float* g = lat + a.r;
  if (a.has_gate) {
    for (int h = tid; h < a.H; h += nt) a.gate[(size_t)t * a.H + h] = 1.f / (1.f + expf(-g[h]));
    g += a.H;
  }
  for (int e = tid; e < a.E; e += nt) a.logits[(size_t)t * a.E + e] = g[e];
  if (a.tiles) {
    const int per = (a.T + a.tn - 1) / a.tn, n = a.H * per;
    for (int i = t * nt + tid; i < n; i += a.T * nt) {
      const int h = i / per, r0 = (i % per) * a.tn;
      a.tiles[i] = make_int4(h, h * a.ldt + r0, min(a.tn, a.T - r0), 0);
    }
    if (t == 0 && tid == 0) *a.n_tiles = n;
  }
}

// ---------------------------------------------------------------- queries through a latent, rotated parts
struct LatentDown {
  const float* proj; int ldp, q_col, kv_col;     // [T, ldp] fp32: q_rank columns from q_col on; r latent, then rot rotated columns from kv_col on
  const float* q_norm; const float* kv_norm;     // [q_rank], [r]
  const float2* rope;                            // [T, rot / 2], neighbouring dimensions turn together
  const int* slot_map;
  int q_rank, ldq, r, rp, rot, rotp, row_stride, n_slots;       // cache row: latent in rp columns, rotated part in the rotp behind them
  float eps; int* status;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_down_kernel(const LatentDown a, T* __restrict__ cq, T* __restrict__ cache) {
  pdl_launch(); pdl_wait();
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x, slot = a.slot_map[t];
  const float* q = a.proj + (size_t)t * a.ldp + a.q_col;
  const float* kv = a.proj + (size_t)t * a.ldp + a.kv_col;
  const bool ok = slot >= 0 && slot < a.n_slots;
  if (!ok && tid == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, t);
  float sq = 0.f, sk = 0.f;
  for (int i = tid; i < a.q_rank; i += nt) sq = fmaf(q[i], q[i], sq);
  for (int i = tid; i < a.r; i += nt) sk = fmaf(kv[i], kv[i], sk);
  const float fq = rsqrtf(block_sum(sq, red) / (float)a.q_rank + a.eps), fk = rsqrtf(block_sum(sk, red) / (float)a.r + a.eps);
  for (int i = tid; i < a.q_rank; i += nt) cq[(size_t)t * a.ldq + i] = to_t<T>(q[i] * fq * a.q_norm[i]);
  if (!ok) return;
  T* dst = cache + (size_t)slot * a.row_stride;
  for (int i = tid; i < a.rp; i += nt) dst[i] = to_t<T>(i < a.r ? kv[i] * fk * a.kv_norm[i] : 0.f);
  for (int i = tid; i < a.rotp; i += nt) {
    float v = 0.f;
    if (i < a.rot) {
      const float2 cs = a.rope[(size_t)t * (a.rot / 2) + i / 2];
      const float x = kv[a.r + i], y = kv[a.r + (i ^ 1)];
      v = i & 1 ? x * cs.x + y * cs.y : x * cs.x - y * cs.y;
    }
    dst[a.rp + i] = to_t<T>(v);
  }
}

struct LatentSplit {
  const float2* rope; int T, ldt, H, d, dp, rot, rotp, ldq;     // rows of H * (d + rot) queries; [H, ldt, dp] and [H, ldt, rotp], whose pads stay as they are
  int4* tiles; int* n_tiles; int tn;
};

template <typename T, int V>
__global__ void __launch_bounds__(256) latent_split_kernel(const LatentSplit a, const T* __restrict__ q, T* __restrict__ qn, T* __restrict__ qr) {
  pdl_launch(); pdl_wait();
  const int t = blockIdx.x, w = a.d + a.rot, tid = threadIdx.x, nt = blockDim.x;
  const T* row = q + (size_t)t * a.ldq;
  const float2* cs = a.rope + (size_t)t * (a.rot / 2);
  for (int i = tid * V; i < a.H * w; i += nt * V) {
    const int h = i / w, j = i % w;
    if constexpr (V == 8) {
      float v[8];
      load8<T>(row + i, v);
      if (j < a.d) { store8<T>(qn + ((size_t)h * a.ldt + t) * a.dp + j, v); continue; }
      const int p = (j - a.d) / 2;
      float o[8];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 c = cs[p + k];
        o[2 * k] = v[2 * k] * c.x - v[2 * k + 1] * c.y; o[2 * k + 1] = v[2 * k + 1] * c.x + v[2 * k] * c.y;
      }
      store8<T>(qr + ((size_t)h * a.ldt + t) * a.rotp + j - a.d, o);
    } else {
      const float x = to_f(row[i]);
      if (j < a.d) { qn[((size_t)h * a.ldt + t) * a.dp + j] = to_t<T>(x); continue; }
      const int r = j - a.d;
      const float2 c = cs[r / 2];
      const float y = to_f(row[i - r + (r ^ 1)]);
      qr[((size_t)h * a.ldt + t) * a.rotp + r] = to_t<T>(r & 1 ? x * c.x + y * c.y : x * c.x - y * c.y);
    }
  }
  if (a.tiles) {
    const int per = (a.T + a.tn - 1) / a.tn, n = a.H * per;
    for (int i = t * nt + tid; i < n; i += a.T * nt) {
      const int h = i / per, r0 = (i % per) * a.tn;
      a.tiles[i] = make_int4(h, h * a.ldt + r0, min(a.tn, a.T - r0), 0);
    }
    if (t == 0 && tid == 0) *a.n_tiles = n;
  }
}

// ---------------------------------------------------------------- absorbed latent attention on the ordinary cores
// One block per (query row, head): scores of a page of keys (a warp takes 16 of them), online softmax, weighted sum of the page's
// latent rows (a thread owns columns tid, tid + 128, ...).
#define LS_COLS 8
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_simt_kernel(const T* __restrict__ q_lat, const T* __restrict__ q_rope, int rotp, const float* __restrict__ sink, const T* __restrict__ cache, const int* __restrict__ page_table,
                                                               const int* __restrict__ kv_len, const int* __restrict__ q_start, const int* __restrict__ q_len,
                                                               const float* __restrict__ gate, T* __restrict__ out, int ldt, int n_seq, int H, int rp,
                                                               int row_stride, int max_pages, int n_slots, float scale, int* status) {
  pdl_launch(); pdl_wait();
  extern __shared__ float qs[];
  __shared__ float sc[64];
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  int seq = -1;
  for (int s = 0; s < n_seq; ++s) if (t >= q_start[s] && t < q_start[s] + q_len[s]) { seq = s; break; }
  if (seq < 0) return;
  const int pos = kv_len[seq] - q_len[seq] + t - q_start[seq];
  const T* qr = q_lat + ((size_t)h * ldt + t) * rp;
  for (int i = tid; i < rp; i += 128) qs[i] = to_f(qr[i]);
  for (int i = tid; i < rotp; i += 128) qs[rp + i] = to_f(q_rope[((size_t)h * ldt + t) * rotp + i]);
  __syncthreads();
  float m = -INFINITY, l = 0.f, o[LS_COLS];
#pragma unroll
  for (int j = 0; j < LS_COLS; ++j) o[j] = 0.f;
  for (int k0 = 0; k0 <= pos; k0 += 64) {
    int slot0 = page_table[(size_t)seq * max_pages + k0 / 64] * 64;
    if (slot0 < 0 || slot0 + 64 > n_slots) { if (tid == 0) ca_dev_fail(status, CA_DEV_BAD_INDEX, t); slot0 = 0; }
    const T* base = cache + (size_t)slot0 * row_stride;
    const int n = min(64, pos + 1 - k0);
    for (int j = warp * 16; j < warp * 16 + 16; ++j) {
      float d = 0.f;
      if (j < n) for (int i = lane; i < rp + rotp; i += 32) d = fmaf(qs[i], to_f(base[(size_t)j * row_stride + i]), d);
      d = warp_sum(d);
      if (lane == 0) sc[j] = j < n ? d * scale : -INFINITY;
    }
    __syncthreads();
    const float s0 = sc[lane], s1 = sc[lane + 32];
    const float mn = fmaxf(m, warp_max(fmaxf(s0, s1)));             // key k0 is visible, so mn is finite
    const float al = m == -INFINITY ? 0.f : expf(m - mn);
    const float p0 = expf(s0 - mn), p1 = expf(s1 - mn);
    l = l * al + warp_sum(p0 + p1);
    m = mn;
    __syncthreads();
    if (warp == 0) { sc[lane] = p0; sc[lane + 32] = p1; }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < LS_COLS; ++c) {
      const int i = tid + c * 128;
      if (i < rp) {
        float acc = o[c] * al;
        for (int j = 0; j < n; ++j) acc = fmaf(sc[j], to_f(base[(size_t)j * row_stride + i]), acc);
        o[c] = acc;
      }
    }
    __syncthreads();
  }
  if (sink) l += expf(sink[h] - m);
  const float f = (l > 0.f ? 1.f / l : 0.f) * (gate ? gate[(size_t)t * H + h] : 1.f);
#pragma unroll
  for (int c = 0; c < LS_COLS; ++c) {
    const int i = tid + c * 128;
    if (i < rp) out[((size_t)h * ldt + t) * rp + i] = to_t<T>(o[c] * f);
  }
}

// ---------------------------------------------------------------- C ABI
struct CaEmit { const float* w; const float* b; void* xn; void* cat; float alpha; int ldn, ldc; int reserved; };

template <typename T>
static Emit<T> emit_from(const CaEmit* e) {
  Emit<T> r = {nullptr, nullptr, 0.f, nullptr, 0, nullptr, 0};
  if (e) { r.w = e->w; r.b = e->b; r.alpha = e->alpha; r.xn = (T*)e->xn; r.ldn = e->ldn; r.cat = (T*)e->cat; r.ldc = e->ldc; }
  return r;
}
static bool emit_ok(const CaEmit* e) { return !e || ((!e->xn || (e->w && e->b && e->ldn % 8 == 0)) && (!e->cat || e->ldc % 8 == 0)); }
static dim3 row_grid(int T, int W) { return dim3(T, (W / 8 + 127) / 128); }

extern "C" int cuteafd_stack_embed(const int* tokens, const int* positions, const void* table, const void* pos_table, float* x, void* x0, int ld0,
                                   int T, int W, int vocab, int n_pos, int f32, const CaEmit* e, int* status, cudaStream_t s) {
  CA_REQUIRE(tokens && positions && table && x && W % 8 == 0 && ld0 % 8 == 0 && emit_ok(e), "stack_embed: bad arguments");
  if (T <= 0) return CA_OK;
  if (f32) CA_LAUNCH_PDL(stack_embed_kernel<float>, row_grid(T, W), 128, 0, s, tokens, positions, (const bf16*)table, (const bf16*)pos_table, x, (float*)x0, ld0, W, vocab, n_pos, status, emit_from<float>(e));
  else CA_LAUNCH_PDL(stack_embed_kernel<bf16>, row_grid(T, W), 128, 0, s, tokens, positions, (const bf16*)table, (const bf16*)pos_table, x, (bf16*)x0, ld0, W, vocab, n_pos, status, emit_from<bf16>(e));
  CA_CHECK_LAUNCH("stack_embed");
  return CA_OK;
}

extern "C" int cuteafd_stack_stream(float* x, const float* vec, const int* src_rows, int T, int W, int f32, const CaEmit* e, cudaStream_t s) {
  CA_REQUIRE(x && W % 8 == 0 && emit_ok(e) && !(vec && src_rows), "stack_stream: bad arguments");
  if (T <= 0) return CA_OK;
  if (f32) CA_LAUNCH_PDL(stack_stream_kernel<float>, row_grid(T, W), 128, 0, s, x, vec, src_rows, W, emit_from<float>(e));
  else CA_LAUNCH_PDL(stack_stream_kernel<bf16>, row_grid(T, W), 128, 0, s, x, vec, src_rows, W, emit_from<bf16>(e));
  CA_CHECK_LAUNCH("stack_stream");
  return CA_OK;
}

extern "C" int cuteafd_stack_combine(float* x, const void* mix, const float* ls1, const void* y, const int* slot_row, const float* wts, const float* ls2,
                                     int T, int W, int k, int f32, const CaEmit* e, cudaStream_t s) {
  CA_REQUIRE(x && mix && ls1 && W % 8 == 0 && emit_ok(e), "stack_combine: bad arguments");
  CA_REQUIRE(k == 0 || (y && slot_row && wts && ls2), "stack_combine: routed rows need their table, weights and scale");
  if (T <= 0) return CA_OK;
  if (f32) CA_LAUNCH_PDL(stack_combine_kernel<float>, row_grid(T, W), 128, 0, s, x, (const float*)mix, ls1, (const float*)y, slot_row, wts, ls2, k, W, emit_from<float>(e));
  else CA_LAUNCH_PDL(stack_combine_kernel<bf16>, row_grid(T, W), 128, 0, s, x, (const bf16*)mix, ls1, (const bf16*)y, slot_row, wts, ls2, k, W, emit_from<bf16>(e));
  CA_CHECK_LAUNCH("stack_combine");
  return CA_OK;
}

extern "C" int cuteafd_latent_prepare(const float* proj, int ldp, const float* norm_w, const int* slot_map, void* q, void* cache, float* gate, float* logits,
                                      void* tiles, int* n_tiles, int T, int ldt, int H, int d, int dp, int r, int rp, int row_stride, int n_slots, int E,
                                      int tn, float eps, int f32, int* status, cudaStream_t s) {
  CA_REQUIRE(proj && norm_w && slot_map && q && cache, "latent_prepare: null argument");
  CA_REQUIRE(H >= 1 && d >= 1 && d <= dp && dp % 8 == 0 && r >= 1 && r <= rp && rp <= row_stride && ldp % 4 == 0 && ldt >= T, "latent_prepare: bad shape");
  CA_REQUIRE(H * d + r + (gate ? H : 0) + E <= ldp && (E == 0 || logits) && (!tiles || (n_tiles && tn >= 1)), "latent_prepare: projection row too short");
  if (T <= 0) return CA_OK;
  LatentPrep a{proj, ldp, norm_w, slot_map, gate, logits, (int4*)tiles, n_tiles, status, T, ldt, H, d, dp, r, rp, row_stride, n_slots, E, tn, gate ? 1 : 0, eps};
  if (f32) CA_LAUNCH_PDL(latent_prepare_kernel<float>, T, 256, 0, s, a, (float*)q, (float*)cache);
  else CA_LAUNCH_PDL(latent_prepare_kernel<bf16>, T, 256, 0, s, a, (bf16*)q, (bf16*)cache);
  CA_CHECK_LAUNCH("latent_prepare");
  return CA_OK;
}

struct CaLatentDown {
  const float* proj; const float* q_norm; const float* kv_norm; const void* rope; const int* slot_map; void* cq; void* cache; int* status;
  int ldp, q_col, kv_col, q_rank, ldq, r, rp, rot, rotp, row_stride, n_slots, T; float eps;
};

extern "C" int cuteafd_latent_down(const CaLatentDown* c, int f32, cudaStream_t s) {
  CA_REQUIRE(c && c->proj && c->q_norm && c->kv_norm && c->slot_map && c->cq && c->cache && (c->rot == 0 || c->rope), "latent_down: null argument");
  CA_REQUIRE(c->q_rank >= 1 && c->q_rank <= c->ldq && c->r >= 1 && c->r <= c->rp && c->rot % 2 == 0 && c->rot <= c->rotp && c->rp + c->rotp <= c->row_stride && c->q_col + c->q_rank <= c->ldp &&
             c->kv_col + c->r + c->rot <= c->ldp && c->q_col >= 0 && c->kv_col >= 0, "latent_down: bad shape");
  if (c->T <= 0) return CA_OK;
  const LatentDown a{c->proj, c->ldp, c->q_col, c->kv_col, c->q_norm, c->kv_norm, (const float2*)c->rope, c->slot_map, c->q_rank, c->ldq, c->r, c->rp, c->rot, c->rotp, c->row_stride,
                     c->n_slots, c->eps, c->status};
  if (f32) CA_LAUNCH_PDL(latent_down_kernel<float>, c->T, 256, 0, s, a, (float*)c->cq, (float*)c->cache);
  else CA_LAUNCH_PDL(latent_down_kernel<bf16>, c->T, 256, 0, s, a, (bf16*)c->cq, (bf16*)c->cache);
  CA_CHECK_LAUNCH("latent_down");
  return CA_OK;
}

extern "C" int cuteafd_latent_split(const void* q, int ldq, const void* rope, void* qn, void* qr, void* tiles, int* n_tiles, int T, int ldt, int H, int d, int dp, int rot, int rotp, int tn,
                                    int f32, cudaStream_t s) {
  CA_REQUIRE(q && qn && (rot == 0 || (rope && qr)) && (!tiles || (n_tiles && tn >= 1)), "latent_split: null argument");
  CA_REQUIRE(H >= 1 && d >= 1 && d <= dp && rot % 2 == 0 && rot >= 0 && rot <= rotp && ldq >= H * (d + rot) && ldt >= T && dp % 8 == 0 && rotp % 8 == 0, "latent_split: bad shape");
  if (T <= 0) return CA_OK;
  const LatentSplit a{(const float2*)rope, T, ldt, H, d, dp, rot, rotp, ldq, (int4*)tiles, n_tiles, tn};
  const bool v8 = ((d | rot | ldq) & 7) == 0 && (((uintptr_t)q | (uintptr_t)qn | (uintptr_t)qr) & 15) == 0;
#define LS_GO(T_, V_) CA_LAUNCH_PDL((latent_split_kernel<T_, V_>), T, 256, 0, s, a, (const T_*)q, (T_*)qn, (T_*)qr)
  if (f32) { if (v8) LS_GO(float, 8); else LS_GO(float, 1); }
  else if (v8) LS_GO(bf16, 8);
  else LS_GO(bf16, 1);
  CA_CHECK_LAUNCH("latent_split");
  return CA_OK;
}

extern "C" int cuteafd_latent_attention_simt(const void* q_lat, const void* q_rope, int rotp, const float* sink, const void* cache, const int* page_table, const int* kv_len, const int* q_start,
                                             const int* q_len, const float* gate, void* out, int T, int ldt, int n_seq, int H, int rp, int row_stride,
                                             int max_pages, int n_slots, float scale, int f32, int* status, cudaStream_t s) {
  CA_REQUIRE(q_lat && cache && page_table && kv_len && q_start && q_len && out, "latent_attention_simt: null argument");
  CA_REQUIRE(H >= 1 && H <= 65535 && rp >= 1 && rp <= 128 * LS_COLS && rotp >= 0 && rotp <= 1024 && (rotp == 0 || q_rope) && rp + rotp <= row_stride && ldt >= T, "latent_attention_simt: latent width %d (at most %d)", rp, 128 * LS_COLS);
  if (T <= 0 || n_seq <= 0) return CA_OK;
  if (f32) CA_LAUNCH_PDL(latent_attn_simt_kernel<float>, dim3(T, H), 128, (rp + rotp) * sizeof(float), s, (const float*)q_lat, (const float*)q_rope, rotp, sink, (const float*)cache, page_table, kv_len, q_start, q_len, gate, (float*)out, ldt, n_seq, H, rp, row_stride, max_pages, n_slots, scale, status);
  else CA_LAUNCH_PDL(latent_attn_simt_kernel<bf16>, dim3(T, H), 128, (rp + rotp) * sizeof(float), s, (const bf16*)q_lat, (const bf16*)q_rope, rotp, sink, (const bf16*)cache, page_table, kv_len, q_start, q_len, gate, (bf16*)out, ldt, n_seq, H, rp, row_stride, max_pages, n_slots, scale, status);
  CA_CHECK_LAUNCH("latent_attention_simt");
  return CA_OK;
}

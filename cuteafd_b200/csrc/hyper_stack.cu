// Kernels of the hyper-connected stacks (several fp32 residual streams mixed by constants at every sub-layer boundary):
//   hyper_embed      token row + row of the pair table (previous token, token) -> every stream, first normalised operand row
//   hyper_add        sub-layer output -> streams: x_t = sum_s mix[s, t] x_s + out[t] y, next sub-layer's input sum_s in[s] x_s, its norm.  y is put
//                    together on the way: bias, the weighted rows of routed experts, or the sum of two mixers' outputs, each normalised
//   hyper_gather     sum of the streams of the rows that need logits, final norm
//   silu_rows        silu(g) * u over two projected rows (all-fp32 mode; bf16 products do it in their epilogue)
// T is the operand type: bf16, or float for the all-fp32 mode.  (No counterpart in the reference, which has no such family; the boundary is the
// constant-coefficient sibling of mhc.cu; their linear mixers are decay_scan.cu's.)
#include "stack_rows.cuh"

#define HY_MAX_STREAMS 8
#define HY_THREADS 512      // most threads of a row

// ---------------------------------------------------------------- residual streams
template <typename T>
struct HyperRows {
  float* x; int S, W, Wp;                                   // [T, S, Wp] residual streams; norms average over W
  const float* next_in;                                     // [S] how the next sub-layer reads the streams
  const float* gain; T* xn; int ldn;                        // next operand: the collapsed row normalised by `gain`, or null
  float eps; int* status;
};

// u holds the collapsed row of this thread's chunks: normalise and hand on.
template <typename T, int NCH>
__device__ __forceinline__ void hyper_emit(const HyperRows<T>& a, float (&u)[NCH][4], size_t row, float* red) {
  if (!a.xn) return;
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NCH; ++c)
#pragma unroll
    for (int j = 0; j < 4; ++j) ss = fmaf(u[c][j], u[c][j], ss);          // pads are zero
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.W + a.eps);
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 4;
    if (i >= a.Wp) continue;
    float g[4], y[4];
    load4<float>(a.gain + i, g);
#pragma unroll
    for (int j = 0; j < 4; ++j) y[j] = u[c][j] * inv * g[j];
    store4<T>(a.xn + row * a.ldn + i, y);
  }
}

struct PairTable {
  const bf16* rows; int buckets; long long mul_prev, mul_cur;       // row (prev * mul_prev + token * mul_cur) mod buckets; row `buckets` starts a sequence
  int* recent; int R;                                       // [slots, R] tokens by position: what the previous steps fed
  const int* state_slot; const int* q_start; const int* q_len; const int* kv_len;
  int n_seq, n_state;
};

template <typename T, int NCH>
__global__ void __launch_bounds__(HY_THREADS, NCH <= 2 ? 2 : 1) hyper_embed_kernel(const HyperRows<T> a, const int* __restrict__ tokens, const bf16* __restrict__ table, int vocab, const PairTable p) {
  pdl_launch(); pdl_wait();
  __shared__ float red[32];
  __shared__ int row_sh;
  const int t = blockIdx.x;
  int tok = tokens[t];
  if (tok < 0 || tok >= vocab) { if (threadIdx.x == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, t); tok = 0; }
  int pair = -1;
  if (p.rows) {
    if (threadIdx.x == 0) row_sh = p.buckets;
    __syncthreads();
    for (int s = threadIdx.x; s < p.n_seq; s += blockDim.x) {
      const int q0 = p.q_start[s], n = p.q_len[s];
      if (t < q0 || t >= q0 + n) continue;
      const int p0 = p.kv_len[s] - n, slot = p.state_slot[s];
      if (slot < 0 || slot >= p.n_state) { ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6F1); continue; }
      int* recent = p.recent + (size_t)slot * p.R;
      int prev = -1;
      if (t > q0) prev = tokens[t - 1];
      else if (p0 > 0) prev = recent[(p0 - 1) % p.R];
      if (prev >= 0) row_sh = (int)(((long long)prev * p.mul_prev + (long long)tok * p.mul_cur) % p.buckets);
      // the run's first row has read what was there: it leaves the run's tokens (the last R of them)
      if (t == q0)
        for (int i = max(0, n - p.R); i < n; ++i) recent[(p0 + i) % p.R] = tokens[q0 + i];
    }
    __syncthreads();
    pair = row_sh;
  }
  float in = 0.f;
  for (int s = 0; s < a.S; ++s) in += a.next_in[s];
  float u[NCH][4];
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j) u[c][j] = 0.f;
    if (i >= a.Wp) continue;
    load4<bf16>(table + (size_t)tok * a.Wp + i, u[c]);
    if (pair >= 0) {
      float b[4];
      load4<bf16>(p.rows + (size_t)pair * a.Wp + i, b);
#pragma unroll
      for (int j = 0; j < 4; ++j) u[c][j] += b[j];
    }
    for (int s = 0; s < a.S; ++s) store4<float>(a.x + ((size_t)t * a.S + s) * a.Wp + i, u[c]);
#pragma unroll
    for (int j = 0; j < 4; ++j) u[c][j] *= in;
  }
  hyper_emit<T, NCH>(a, u, t, red);
}

template <typename T>
struct SubOutput {                                          // what a sub-layer leaves: y = sa * A + sb * B + routed
  const T* a; const T* b; const float* bias;                // rows Wp apart (either may be null); bias is added to A
  const float* ga; const float* gb; float sa, sb;           // gains of norms over A and B (null: none)
  const T* y; const int* slot_row; const float* wts; int k; // routed experts' rows: sum of wts * y[slot_row] over the token's k routes
  const float* out; const float* mix;                       // [S], [S, S] from the closing sub-layer's constants
};

// PAIR: two outputs (B and its norm); otherwise A and routed rows alone.
template <typename T, int SM, int NCH, bool PAIR>
__global__ void __launch_bounds__(HY_THREADS, NCH <= 2 ? 2 : 1) hyper_add_kernel(const HyperRows<T> a, const SubOutput<T> o) {
  pdl_launch(); pdl_wait();
  __shared__ float red[32];
  __shared__ float mix[SM * SM], out[SM], in[SM];
  const int t = blockIdx.x, S = SM <= 4 ? SM : a.S;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) mix[i] = o.mix[i];
  if ((int)threadIdx.x < S) { out[threadIdx.x] = o.out[threadIdx.x]; in[threadIdx.x] = a.next_in ? a.next_in[threadIdx.x] : 0.f; }
  constexpr int NZ = PAIR ? NCH : 1;
  float y[NCH][4], z[NZ][4], sy = 0.f, sz = 0.f;
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j) { y[c][j] = 0.f; if (PAIR) z[c % NZ][j] = 0.f; }
    if (i >= a.Wp) continue;
    if (o.a) load4<T>(o.a + (size_t)t * a.Wp + i, y[c]);
    if (PAIR) load4<T>(o.b + (size_t)t * a.Wp + i, z[c % NZ]);
    if (o.bias) {
      float b[4];
      load4<float>(o.bias + i, b);
#pragma unroll
      for (int j = 0; j < 4; ++j) y[c][j] += b[j];
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) { sy = fmaf(y[c][j], y[c][j], sy); if (PAIR) sz = fmaf(z[c % NZ][j], z[c % NZ][j], sz); }
  }
  const float fy = o.sa * (o.ga ? rsqrtf(block_sum(sy, red) / (float)a.W + a.eps) : 1.f);
  const float fz = !PAIR ? 0.f : o.sb * (o.gb ? rsqrtf(block_sum(sz, red) / (float)a.W + a.eps) : 1.f);
  __syncthreads();                                          // mix, out and in are there
  float u[NCH][4];
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j) u[c][j] = 0.f;
    if (i >= a.Wp) continue;
    float g[4] = {1.f, 1.f, 1.f, 1.f}, h[4] = {1.f, 1.f, 1.f, 1.f};
    if (o.ga) load4<float>(o.ga + i, g);
    if (PAIR && o.gb) load4<float>(o.gb + i, h);
#pragma unroll
    for (int j = 0; j < 4; ++j) y[c][j] = fy * y[c][j] * g[j] + (PAIR ? fz * z[c % NZ][j] * h[j] : 0.f);
    // four routes at a time: row numbers and weights first, then all rows in flight together
    for (int r0 = 0; r0 < o.k; r0 += 4) {
      int r[4]; float w[4], q[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const bool live = r0 + j < o.k;
        r[j] = live ? o.slot_row[(size_t)t * o.k + r0 + j] : -1; w[j] = live ? o.wts[(size_t)t * o.k + r0 + j] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) if (r[j] >= 0) load4<T>(o.y + (size_t)r[j] * a.Wp + i, q[j]);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (r[j] >= 0) {
#pragma unroll
          for (int e = 0; e < 4; ++e) y[c][e] = fmaf(w[j], q[j][e], y[c][e]);
        }
    }
    float* x = a.x + (size_t)t * a.S * a.Wp + i;
    float v[SM][4];
#pragma unroll
    for (int s = 0; s < SM; ++s) if (s < S) load4<float>(x + (size_t)s * a.Wp, v[s]);
#pragma unroll
    for (int d = 0; d < SM; ++d)
      if (d < S) {
        float n[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) n[j] = out[d] * y[c][j];
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < S) {
#pragma unroll
            for (int j = 0; j < 4; ++j) n[j] = fmaf(mix[s * S + d], v[s][j], n[j]);
          }
        store4<float>(x + (size_t)d * a.Wp, n);
#pragma unroll
        for (int j = 0; j < 4; ++j) u[c][j] = fmaf(in[d], n[j], u[c][j]);
      }
  }
  hyper_emit<T, NCH>(a, u, t, red);
}

template <typename T, int NCH>
__global__ void __launch_bounds__(HY_THREADS, NCH <= 2 ? 2 : 1) hyper_gather_kernel(const HyperRows<T> a, const int* __restrict__ src_rows) {
  pdl_launch(); pdl_wait();
  __shared__ float red[32];
  const size_t row = src_rows[blockIdx.x];
  float u[NCH][4];
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j) u[c][j] = 0.f;
    if (i >= a.Wp) continue;
    for (int s = 0; s < a.S; ++s) {
      float v[4];
      load4<float>(a.x + (row * a.S + s) * a.Wp + i, v);
#pragma unroll
      for (int j = 0; j < 4; ++j) u[c][j] += v[j];
    }
  }
  hyper_emit<T, NCH>(a, u, blockIdx.x, red);
}

// ---------------------------------------------------------------- silu(g) * u over two projected rows
template <typename T>
__global__ void silu_rows_kernel(const T* __restrict__ g, const T* __restrict__ u, T* __restrict__ out, int ldi, int ldo, int N) {
  pdl_launch(); pdl_wait();
  const size_t t = blockIdx.x;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < N; i += gridDim.y * blockDim.x) {
    const float z = to_f(g[t * ldi + i]);
    out[t * ldo + i] = to_t<T>(z / (1.f + expf(-z)) * to_f(u[t * ldi + i]));
  }
}

// ---------------------------------------------------------------- C ABI
struct CaHyperRows {
  float* x; const float* next_in; const float* gain; void* xn; int* status;
  const int* tokens; const void* table; const void* pair_rows; int* recent; const int* state_slot; const int* q_start; const int* q_len; const int* kv_len;      // embed
  const void* a; const void* b; const float* bias; const float* ga; const float* gb; const void* y; const int* slot_row; const float* wts; const float* out; const float* mix;  // add
  const int* src_rows;                                                                                                                                            // gather
  long long mul_prev, mul_cur;
  int S, W, Wp, ldn, vocab, buckets, R, n_seq, n_state, k; float eps, sa, sb;
};
enum { HYPER_EMBED = 0, HYPER_ADD = 1, HYPER_GATHER = 2 };

template <typename T, int NCH>
static int hyper_launch(const CaHyperRows* c, int mode, int rows, int nt, cudaStream_t s) {
  const HyperRows<T> a{c->x, c->S, c->W, c->Wp, c->next_in, c->gain, (T*)c->xn, c->ldn, c->eps, c->status};
  if (mode == HYPER_EMBED) {
    const PairTable p{(const bf16*)c->pair_rows, c->buckets, c->mul_prev, c->mul_cur, c->recent, c->R, c->state_slot, c->q_start, c->q_len, c->kv_len, c->n_seq, c->n_state};
    CA_LAUNCH_PDL((hyper_embed_kernel<T, NCH>), rows, nt, 0, s, a, c->tokens, (const bf16*)c->table, c->vocab, p);
  } else if (mode == HYPER_GATHER) {
    CA_LAUNCH_PDL((hyper_gather_kernel<T, NCH>), rows, nt, 0, s, a, c->src_rows);
  } else {
    const SubOutput<T> o{(const T*)c->a, (const T*)c->b, c->bias, c->ga, c->gb, c->sa, c->sb, (const T*)c->y, c->slot_row, c->wts, c->k, c->out, c->mix};
#define HY_ADD(SM_)                                                                                  \
    if (c->b) CA_LAUNCH_PDL((hyper_add_kernel<T, SM_, NCH, true>), rows, nt, 0, s, a, o);            \
    else CA_LAUNCH_PDL((hyper_add_kernel<T, SM_, NCH, false>), rows, nt, 0, s, a, o);
    if (c->S == 1) { HY_ADD(1) } else if (c->S == 2) { HY_ADD(2) } else if (c->S == 3) { HY_ADD(3) } else if (c->S == 4) { HY_ADD(4) } else { HY_ADD(HY_MAX_STREAMS) }
  }
  CA_CHECK_LAUNCH("hyper_rows");
  return CA_OK;
}

extern "C" int cuteafd_hyper_rows(const CaHyperRows* c, int mode, int rows, int f32, cudaStream_t s) {
  CA_REQUIRE(c && c->x && c->S >= 1 && c->S <= HY_MAX_STREAMS && c->W >= 1 && c->Wp >= c->W && c->Wp % 8 == 0 && c->Wp <= 64 * HY_THREADS, "hyper_rows: 1 to %d streams of up to %d values", HY_MAX_STREAMS, 64 * HY_THREADS);
  CA_REQUIRE(!c->xn || (c->gain && c->ldn % 8 == 0 && c->ldn >= c->Wp && (mode == HYPER_GATHER || c->next_in)), "hyper_rows: next operand without its norm or stream weights");
  if (mode == HYPER_EMBED) {
    CA_REQUIRE(c->tokens && c->table && c->vocab > 0 && c->next_in, "hyper_rows: embedding without tokens or table");
    CA_REQUIRE(!c->pair_rows || (c->buckets >= 1 && c->recent && c->R >= 1 && c->state_slot && c->q_start && c->q_len && c->kv_len && c->mul_prev >= 0 && c->mul_cur >= 0), "hyper_rows: pair table without its sequences");
  } else if (mode == HYPER_ADD) {
    CA_REQUIRE(c->out && c->mix && (c->k == 0 || (c->y && c->slot_row && c->wts)) && (!c->gb || c->b) && (!c->ga || c->a), "hyper_rows: incomplete sub-layer output");
  } else {
    CA_REQUIRE(mode == HYPER_GATHER && c->src_rows && c->xn, "hyper_rows: mode %d without its inputs", mode);
  }
  if (rows <= 0) return CA_OK;
  // four values a thread and chunk; the fewest chunks that HY_THREADS threads cover
  const int pieces = c->Wp / 4, nch = pieces <= HY_THREADS ? 1 : (pieces <= 2 * HY_THREADS ? 2 : (pieces <= 4 * HY_THREADS ? 4 : 16));
  const int nt = ((pieces + nch - 1) / nch + 31) / 32 * 32;
  if (nch == 1) return f32 ? hyper_launch<float, 1>(c, mode, rows, nt, s) : hyper_launch<bf16, 1>(c, mode, rows, nt, s);
  if (nch == 2) return f32 ? hyper_launch<float, 2>(c, mode, rows, nt, s) : hyper_launch<bf16, 2>(c, mode, rows, nt, s);
  if (nch == 4) return f32 ? hyper_launch<float, 4>(c, mode, rows, nt, s) : hyper_launch<bf16, 4>(c, mode, rows, nt, s);
  return f32 ? hyper_launch<float, 16>(c, mode, rows, nt, s) : hyper_launch<bf16, 16>(c, mode, rows, nt, s);
}

extern "C" int cuteafd_silu_rows(const void* g, const void* u, void* out, int T, int ldi, int ldo, int N, int f32, cudaStream_t s) {
  CA_REQUIRE(g && u && out && N >= 1 && ldi >= N && ldo >= N, "silu_rows: bad arguments");
  if (T <= 0) return CA_OK;
  const dim3 grid(T, (N + 1023) / 1024);
  if (f32) CA_LAUNCH_PDL(silu_rows_kernel<float>, grid, 256, 0, s, (const float*)g, (const float*)u, (float*)out, ldi, ldo, N);
  else CA_LAUNCH_PDL(silu_rows_kernel<bf16>, grid, 256, 0, s, (const bf16*)g, (const bf16*)u, (bf16*)out, ldi, ldo, N);
  CA_CHECK_LAUNCH("silu_rows");
  return CA_OK;
}

// Kernels of the hyper-connected stacks (several fp32 residual streams mixed by constants at every sub-layer boundary):
//   hyper_embed      token row + row of the pair table (previous token, token) -> every stream, first normalised operand row
//   hyper_add        sub-layer output -> streams: x_t = sum_s mix[s, t] x_s + out[t] y, next sub-layer's input sum_s in[s] x_s, its norm.  y is put
//                    together on the way: bias, the weighted rows of routed experts, or the sum of two mixers' outputs, each normalised
//   hyper_gather     sum of the streams of the rows that need logits, final norm
//   decay_scan       linear attention with a decay (one constant per head, or one per key channel and token): rotation, decays, recurrence, output
//                    norm, gate; any run length, the state crosses HBM once per 16 tokens
//   silu_rows        silu(g) * u over two projected rows (all-fp32 mode; bf16 products do it in their epilogue)
// T is the operand type: bf16, or float for the all-fp32 mode.  (No counterpart in the reference, which has no such family; the boundary is
// the constant-coefficient sibling of mhc.cu, the recurrence of linear_attn.cu.)
#include "stack_rows.cuh"

#define HY_MAX_STREAMS 8

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
__device__ __forceinline__ void hyper_emit(const HyperRows<T>& a, float (&u)[NCH][8], size_t row, float* red) {
  if (!a.xn) return;
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NCH; ++c)
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(u[c][j], u[c][j], ss);          // pads are zero
  const float inv = rsqrtf(block_sum(ss, red) / (float)a.W + a.eps);
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 8;
    if (i >= a.Wp) continue;
    float g[8], y[8];
    load8<float>(a.gain + i, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) y[j] = u[c][j] * inv * g[j];
    store8<T>(a.xn + row * a.ldn + i, y);
  }
}

struct PairTable {
  const bf16* rows; int buckets; long long mul_prev, mul_cur;       // row (prev * mul_prev + token * mul_cur) mod buckets; row `buckets` starts a sequence
  int* recent; int R;                                       // [slots, R] tokens by position: what the previous steps fed
  const int* state_slot; const int* q_start; const int* q_len; const int* kv_len;
  int n_seq, n_state;
};

template <typename T, int NCH>
__global__ void hyper_embed_kernel(const HyperRows<T> a, const int* __restrict__ tokens, const bf16* __restrict__ table, int vocab, const PairTable p) {
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
  float u[NCH][8];
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) u[c][j] = 0.f;
    if (i >= a.Wp) continue;
    load8<bf16>(table + (size_t)tok * a.Wp + i, u[c]);
    if (pair >= 0) {
      float b[8];
      load8<bf16>(p.rows + (size_t)pair * a.Wp + i, b);
#pragma unroll
      for (int j = 0; j < 8; ++j) u[c][j] += b[j];
    }
    for (int s = 0; s < a.S; ++s) store8<float>(a.x + ((size_t)t * a.S + s) * a.Wp + i, u[c]);
#pragma unroll
    for (int j = 0; j < 8; ++j) u[c][j] *= in;
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

template <typename T, int SM, int NCH>
__global__ void hyper_add_kernel(const HyperRows<T> a, const SubOutput<T> o) {
  pdl_launch(); pdl_wait();
  __shared__ float red[32];
  __shared__ float mix[SM * SM], out[SM], in[SM];
  const int t = blockIdx.x, S = SM <= 4 ? SM : a.S;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) mix[i] = o.mix[i];
  if ((int)threadIdx.x < S) { out[threadIdx.x] = o.out[threadIdx.x]; in[threadIdx.x] = a.next_in ? a.next_in[threadIdx.x] : 0.f; }
  float y[NCH][8], z[NCH][8], sy = 0.f, sz = 0.f;
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) y[c][j] = z[c][j] = 0.f;
    if (i >= a.Wp) continue;
    if (o.a) load8<T>(o.a + (size_t)t * a.Wp + i, y[c]);
    if (o.b) load8<T>(o.b + (size_t)t * a.Wp + i, z[c]);
    if (o.bias) {
      float b[8];
      load8<float>(o.bias + i, b);
#pragma unroll
      for (int j = 0; j < 8; ++j) y[c][j] += b[j];
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) { sy = fmaf(y[c][j], y[c][j], sy); sz = fmaf(z[c][j], z[c][j], sz); }
  }
  const float fy = o.sa * (o.ga ? rsqrtf(block_sum(sy, red) / (float)a.W + a.eps) : 1.f);
  const float fz = o.sb * (o.gb ? rsqrtf(block_sum(sz, red) / (float)a.W + a.eps) : 1.f);
  __syncthreads();                                          // mix, out and in are there
  float u[NCH][8];
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) u[c][j] = 0.f;
    if (i >= a.Wp) continue;
    float g[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f}, h[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
    if (o.ga) load8<float>(o.ga + i, g);
    if (o.gb) load8<float>(o.gb + i, h);
#pragma unroll
    for (int j = 0; j < 8; ++j) y[c][j] = fy * y[c][j] * g[j] + fz * z[c][j] * h[j];
    // eight routes at a time: row numbers and weights first, then all rows in flight together
    for (int r0 = 0; r0 < o.k; r0 += 8) {
      int r[8]; float w[8], q[8][8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const bool live = r0 + j < o.k;
        r[j] = live ? o.slot_row[(size_t)t * o.k + r0 + j] : -1; w[j] = live ? o.wts[(size_t)t * o.k + r0 + j] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) if (r[j] >= 0) load8<T>(o.y + (size_t)r[j] * a.Wp + i, q[j]);
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (r[j] >= 0) {
#pragma unroll
          for (int e = 0; e < 8; ++e) y[c][e] = fmaf(w[j], q[j][e], y[c][e]);
        }
    }
    float* x = a.x + (size_t)t * a.S * a.Wp + i;
    float v[SM][8];
#pragma unroll
    for (int s = 0; s < SM; ++s) if (s < S) load8<float>(x + (size_t)s * a.Wp, v[s]);
#pragma unroll
    for (int d = 0; d < SM; ++d)
      if (d < S) {
        float n[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) n[j] = out[d] * y[c][j];
#pragma unroll
        for (int s = 0; s < SM; ++s)
          if (s < S) {
#pragma unroll
            for (int j = 0; j < 8; ++j) n[j] = fmaf(mix[s * S + d], v[s][j], n[j]);
          }
        store8<float>(x + (size_t)d * a.Wp, n);
#pragma unroll
        for (int j = 0; j < 8; ++j) u[c][j] = fmaf(in[d], n[j], u[c][j]);
      }
  }
  hyper_emit<T, NCH>(a, u, t, red);
}

template <typename T, int NCH>
__global__ void hyper_gather_kernel(const HyperRows<T> a, const int* __restrict__ src_rows) {
  pdl_launch(); pdl_wait();
  __shared__ float red[32];
  const size_t row = src_rows[blockIdx.x];
  float u[NCH][8];
#pragma unroll
  for (int c = 0; c < NCH; ++c) {
    const int i = (threadIdx.x + c * blockDim.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) u[c][j] = 0.f;
    if (i >= a.Wp) continue;
    for (int s = 0; s < a.S; ++s) {
      float v[8];
      load8<float>(a.x + (row * a.S + s) * a.Wp + i, v);
#pragma unroll
      for (int j = 0; j < 8; ++j) u[c][j] += v[j];
    }
  }
  hyper_emit<T, NCH>(a, u, blockIdx.x, red);
}

// ---------------------------------------------------------------- linear attention with a decay
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   out_t = norm(o_t) * silu(g_t)
// A state slot holds two states per head, each with the position it belongs to (-1: the zero state in front of a sequence).  A run starts from
// the state right in front of it and leaves its last state in the other place, so a repeated step repeats its writes.  Runs of up to `depth`
// tokens also leave their keys, decays and values (`ring`, by position): when some of them are taken back, the next run starts from the
// earlier state and absorbs the kept ones again.
#define DS_THREADS 256
#define DS_GROUP 16         // tokens of one pass over the state (at least 2 depth - 1)
#define DS_ROWS 4           // state rows a thread has in flight

template <typename T>
struct DecayScan {
  const T* q; const T* k; const T* v; const T* g; int ldp;  // column views of the projection rows: [H * dim], [H * dim], [H * vdim], [H * vdim]
  const float2* rope; int pairs;                            // [T, pairs], dimensions i and i + pairs turn together; null = none
  float q_scale, k_scale;
  const float* decay;                                       // [H] constant decays; null: alpha = sigmoid(a2 a1 + a2_b)^(1 / tau) per key channel
  const T* a1; const float* a2; const float* a2_b;          // [rank] columns of the projection rows, [H * dim, rank], [H * dim]
  int rank; float inv_tau;
  const float* norm; float eps, out_scale;                  // gain of the output norm [vdim], or null
  float* state; int* tags; float* ring;                     // [slots, 2, H, dim, vp], [slots, H, 2], [slots, depth, H, 2 dim + vp]
  const int* state_slot; const int* q_start; const int* q_len; const int* kv_len;
  T* out; int ldo;
  int H, dim, vdim, vp, depth, n_state;
  int* status;
};

// log alpha of a channel from its logit
__device__ __forceinline__ float log_decay(float z, float inv_tau) { return -(fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))) * inv_tau; }

struct ScanBase { int place, pos, replay; };               // where a run starts: which of the two states, its position, tokens to absorb again
__device__ __forceinline__ ScanBase scan_base(const int* tags, int p0) {
  if (p0 == 0) return ScanBase{0, -1, 0};
  const int c0 = tags[0] < p0 ? tags[0] : -2, c1 = tags[1] < p0 ? tags[1] : -2;
  const int pos = max(c0, c1);
  return ScanBase{c1 > c0 ? 1 : 0, pos, p0 - 1 - pos};
}

struct ScanTile { float* q; float* k; float* al; float* v; float* red; float* o; };

// One pass over the state for `cnt` (<= NT) tokens of the tile, the first `replay` of which only advance it; partial outputs of this thread's
// rows stay in acc.
template <int NT>
__device__ __forceinline__ void scan_pass(const ScanTile& sm, const float* src, float* dst, float* mid, int cnt, int replay, int dim, int vp, int rg, int RG, int c4, float4 (&acc)[NT]) {
#pragma unroll
  for (int t = 0; t < NT; ++t) acc[t] = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int r0 = rg; r0 < dim; r0 += RG * DS_ROWS) {
    float4 S[DS_ROWS];
#pragma unroll
    for (int i = 0; i < DS_ROWS; ++i) {
      const int r = r0 + i * RG;
      S[i] = src && r < dim ? *(const float4*)(src + (size_t)r * vp + c4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      if (t >= cnt) break;
      const float4 v = *(const float4*)(sm.v + t * vp + c4);
#pragma unroll
      for (int i = 0; i < DS_ROWS; ++i) {
        const int r = min(r0 + i * RG, dim - 1);
        const float al = sm.al[t * dim + r], k = sm.k[t * dim + r], q = sm.q[t * dim + r];
        S[i].x = fmaf(al, S[i].x, k * v.x); S[i].y = fmaf(al, S[i].y, k * v.y); S[i].z = fmaf(al, S[i].z, k * v.z); S[i].w = fmaf(al, S[i].w, k * v.w);
        if (r0 + i * RG < dim) {
          acc[t].x = fmaf(q, S[i].x, acc[t].x); acc[t].y = fmaf(q, S[i].y, acc[t].y); acc[t].z = fmaf(q, S[i].z, acc[t].z); acc[t].w = fmaf(q, S[i].w, acc[t].w);
        }
      }
      if (mid && t == replay - 1) {
#pragma unroll
        for (int i = 0; i < DS_ROWS; ++i) if (r0 + i * RG < dim) *(float4*)(mid + (size_t)(r0 + i * RG) * vp + c4) = S[i];
      }
    }
#pragma unroll
    for (int i = 0; i < DS_ROWS; ++i) if (r0 + i * RG < dim) *(float4*)(dst + (size_t)(r0 + i * RG) * vp + c4) = S[i];
  }
}

template <typename T>
__global__ void __launch_bounds__(DS_THREADS) decay_scan_kernel(const DecayScan<T> a, int cap) {
  pdl_launch(); pdl_wait();
  extern __shared__ float ds_smem[];
  __shared__ float red32[32];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, dim = a.dim, vp = a.vp;
  const int n = a.q_len[seq], p0 = a.kv_len[seq] - n, row0 = a.q_start[seq], slot = a.state_slot[seq];
  if (n <= 0) return;
  if (slot < 0 || slot >= a.n_state) { if (tid == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6F2); return; }
  ScanTile sm;
  sm.q = ds_smem; sm.k = sm.q + cap * dim; sm.al = sm.k + cap * dim; sm.v = sm.al + cap * dim; sm.red = sm.v + cap * vp; sm.o = sm.red + 4 * DS_THREADS;
  int* tags = a.tags + ((size_t)slot * a.H + h) * 2;
  const ScanBase b = scan_base(tags, p0);
  if (b.pos < -1 || b.replay >= a.depth) { if (tid == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6F3); return; }
  const size_t one = (size_t)dim * vp;
  float* base = a.state + (((size_t)slot * 2 + b.place) * a.H + h) * one;
  float* last = a.state + (((size_t)slot * 2 + 1 - b.place) * a.H + h) * one;
  const int rw = 2 * dim + vp;
  float* ring = a.ring + ((size_t)slot * a.depth * a.H + h) * rw;           // entry of position p: + (p % depth) * H * rw
  const int CG = vp / 4, RG = DS_THREADS / CG, c4 = (tid % CG) * 4, rg = tid / CG;
  const bool works = rg < RG;
  const float decay = a.decay ? a.decay[h] : 0.f;

  for (int done = 0, first = 1; first || done < n; first = 0) {
    const int replay = first ? b.replay : 0, cnt = min(cap, replay + n - done), fresh = cnt - replay;
    __syncthreads();
    for (int i = tid; i < cnt * dim; i += DS_THREADS) {
      const int t = i / dim, r = i % dim;
      if (t < replay) {
        const float* e = ring + (size_t)((b.pos + 1 + t) % a.depth) * a.H * rw;
        sm.k[i] = e[r]; sm.al[i] = e[dim + r]; sm.q[i] = 0.f;
        continue;
      }
      const int row = row0 + done + t - replay;
      const T* qr = a.q + (size_t)row * a.ldp + h * dim;
      const T* kr = a.k + (size_t)row * a.ldp + h * dim;
      float q = to_f(qr[r]), k = to_f(kr[r]);
      if (a.rope && r < 2 * a.pairs) {
        const bool lo = r < a.pairs;
        const int pr = lo ? r : r - a.pairs, o = lo ? r + a.pairs : pr;
        const float2 cs = a.rope[(size_t)row * a.pairs + pr];
        const float q2 = to_f(qr[o]), k2 = to_f(kr[o]);
        q = lo ? q * cs.x - q2 * cs.y : q * cs.x + q2 * cs.y;
        k = lo ? k * cs.x - k2 * cs.y : k * cs.x + k2 * cs.y;
      }
      float al = decay;
      if (!a.decay) {
        float z = a.a2_b[h * dim + r];
        const T* ar = a.a1 + (size_t)row * a.ldp;
        const float* wr = a.a2 + (size_t)(h * dim + r) * a.rank;
        for (int j = 0; j < a.rank; ++j) z = fmaf(wr[j], to_f(ar[j]), z);
        al = expf(log_decay(z, a.inv_tau));
      }
      sm.q[i] = q * a.q_scale; sm.k[i] = k * a.k_scale; sm.al[i] = al;
    }
    for (int i = tid; i < cnt * vp; i += DS_THREADS) {
      const int t = i / vp, c = i % vp;
      if (t < replay) sm.v[i] = ring[(size_t)((b.pos + 1 + t) % a.depth) * a.H * rw + 2 * dim + c];
      else sm.v[i] = c < a.vdim ? to_f(a.v[(size_t)(row0 + done + t - replay) * a.ldp + h * a.vdim + c]) : 0.f;
    }
    __syncthreads();                                        // the tile is there, and the ring entries that were needed have been read
    if (n >= 2 && n <= a.depth) {
      for (int i = tid; i < fresh * rw; i += DS_THREADS) {
        const int t = i / rw, c = i % rw, s = replay + t;
        ring[(size_t)((p0 + t) % a.depth) * a.H * rw + c] = c < dim ? sm.k[s * dim + c] : (c < 2 * dim ? sm.al[s * dim + c - dim] : sm.v[s * vp + c - 2 * dim]);
      }
    }
    const float* src = first ? (b.pos >= 0 ? base : nullptr) : last;
    float* mid = replay ? base : nullptr;
    // outputs of one token: sum over the row groups, norm, gate
    auto finish = [&](int t, const float4& part) {
      __syncthreads();
      if (works) *(float4*)(sm.red + rg * vp + c4) = part;
      __syncthreads();
      float ss = 0.f;
      for (int c = tid; c < a.vdim; c += DS_THREADS) {
        float o = 0.f;
        for (int g = 0; g < RG; ++g) o += sm.red[g * vp + c];
        sm.o[c] = o;
        ss = fmaf(o, o, ss);
      }
      const float inv = rsqrtf(block_sum(ss, red32) / (float)a.vdim + a.eps) * a.out_scale;
      const size_t row = row0 + done + t - replay;
      for (int c = tid; c < a.vdim; c += DS_THREADS) {
        const float g = to_f(a.g[row * a.ldp + h * a.vdim + c]);
        a.out[row * a.ldo + h * a.vdim + c] = to_t<T>(sm.o[c] * inv * (a.norm ? a.norm[c] : 1.f) * (g / (1.f + expf(-g))));
      }
    };
    if (cnt == 1) {
      float4 acc[1];
      if (works) scan_pass<1>(sm, src, last, mid, cnt, replay, dim, vp, rg, RG, c4, acc);
      finish(0, acc[0]);
    } else {
      float4 acc[DS_GROUP];
      if (works) scan_pass<DS_GROUP>(sm, src, last, mid, cnt, replay, dim, vp, rg, RG, c4, acc);
#pragma unroll
      for (int t = 0; t < DS_GROUP; ++t) if (t >= replay && t < cnt) finish(t, acc[t]);
    }
    done += fresh;
  }
  if (tid == 0) {
    tags[b.place] = b.replay ? p0 - 1 : b.pos;
    tags[1 - b.place] = p0 + n - 1;
  }
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
    if (c->S == 1) CA_LAUNCH_PDL((hyper_add_kernel<T, 1, NCH>), rows, nt, 0, s, a, o);
    else if (c->S == 2) CA_LAUNCH_PDL((hyper_add_kernel<T, 2, NCH>), rows, nt, 0, s, a, o);
    else if (c->S == 3) CA_LAUNCH_PDL((hyper_add_kernel<T, 3, NCH>), rows, nt, 0, s, a, o);
    else if (c->S == 4) CA_LAUNCH_PDL((hyper_add_kernel<T, 4, NCH>), rows, nt, 0, s, a, o);
    else CA_LAUNCH_PDL((hyper_add_kernel<T, HY_MAX_STREAMS, NCH>), rows, nt, 0, s, a, o);
  }
  CA_CHECK_LAUNCH("hyper_rows");
  return CA_OK;
}

extern "C" int cuteafd_hyper_rows(const CaHyperRows* c, int mode, int rows, int f32, cudaStream_t s) {
  CA_REQUIRE(c && c->x && c->S >= 1 && c->S <= HY_MAX_STREAMS && c->W >= 1 && c->Wp >= c->W && c->Wp % 8 == 0 && c->Wp <= 65536, "hyper_rows: 1 to %d streams of up to 65536 values", HY_MAX_STREAMS);
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
  const int chunks = c->Wp / 8, nt = chunks <= 1024 ? (chunks + 31) / 32 * 32 : 1024;
  if (chunks <= 1024) return f32 ? hyper_launch<float, 1>(c, mode, rows, nt, s) : hyper_launch<bf16, 1>(c, mode, rows, nt, s);
  if (chunks <= 2048) return f32 ? hyper_launch<float, 2>(c, mode, rows, nt, s) : hyper_launch<bf16, 2>(c, mode, rows, nt, s);
  return f32 ? hyper_launch<float, 8>(c, mode, rows, nt, s) : hyper_launch<bf16, 8>(c, mode, rows, nt, s);
}

struct CaDecayScan {
  const void* q; const void* k; const void* v; const void* g; const void* rope; const float* decay; const void* a1; const float* a2; const float* a2_b; const float* norm;
  float* state; int* tags; float* ring; const int* state_slot; const int* q_start; const int* q_len; const int* kv_len; void* out; int* status;
  int ldp, pairs, rank, ldo, H, dim, vdim, vp, depth, n_state, n_seq, max_q_len; float q_scale, k_scale, inv_tau, eps, out_scale;
};

template <typename T>
static DecayScan<T> decay_scan_args(const CaDecayScan* c) {
  return DecayScan<T>{(const T*)c->q, (const T*)c->k, (const T*)c->v, (const T*)c->g, c->ldp, (const float2*)c->rope, c->pairs, c->q_scale, c->k_scale, c->decay, (const T*)c->a1, c->a2,
                      c->a2_b, c->rank, c->inv_tau, c->norm, c->eps, c->out_scale, c->state, c->tags, c->ring, c->state_slot, c->q_start, c->q_len, c->kv_len, (T*)c->out, c->ldo,
                      c->H, c->dim, c->vdim, c->vp, c->depth, c->n_state, c->status};
}

template <typename T>
static int decay_scan_launch(const CaDecayScan* c, cudaStream_t s) {
  const int cap = c->max_q_len + c->depth - 1 < DS_GROUP ? c->max_q_len + c->depth - 1 : DS_GROUP;
  const size_t smem = ((size_t)cap * (3 * c->dim + c->vp) + 4 * DS_THREADS + c->vp) * sizeof(float);
  static bool attr_set[64] = {false};
  int dev = 0; cudaGetDevice(&dev);
  if (!attr_set[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(decay_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return ca_cuda(e, "cudaFuncSetAttribute(decay_scan)");
    attr_set[dev & 63] = true;
  }
  CA_REQUIRE(smem <= 200 * 1024, "decay_scan: heads of %d x %d do not fit shared memory", c->dim, c->vdim);
  CA_LAUNCH_PDL((decay_scan_kernel<T>), dim3(c->H, c->n_seq), DS_THREADS, smem, s, decay_scan_args<T>(c), cap);
  CA_CHECK_LAUNCH("decay_scan");
  return CA_OK;
}

extern "C" int cuteafd_decay_scan(const CaDecayScan* c, int f32, cudaStream_t s) {
  CA_REQUIRE(c && c->q && c->k && c->v && c->g && c->state && c->tags && c->ring && c->state_slot && c->q_start && c->q_len && c->kv_len && c->out, "decay_scan: null argument");
  CA_REQUIRE(c->decay || (c->a1 && c->a2 && c->a2_b && c->rank >= 1), "decay_scan: neither constant decays nor a projection of them");
  CA_REQUIRE(c->H >= 1 && c->dim >= 1 && c->dim <= 512 && c->vdim >= 1 && c->vp % 4 == 0 && c->vp >= c->vdim && c->vp <= 4 * DS_THREADS, "decay_scan: heads of %d x %d (at most 512 x %d)", c->dim, c->vdim, 4 * DS_THREADS);
  CA_REQUIRE(c->pairs >= 0 && 2 * c->pairs <= c->dim && (c->pairs == 0 || c->rope) && c->depth >= 1 && 2 * c->depth - 1 <= DS_GROUP && c->n_state >= 1, "decay_scan: bad rotation or depth");
  CA_REQUIRE(c->ldo >= c->H * c->vdim && c->ldp >= c->H * c->vdim && c->ldp >= c->H * c->dim, "decay_scan: rows too short");
  if (c->n_seq <= 0 || c->max_q_len <= 0) return CA_OK;
  CA_REQUIRE(c->n_seq <= 65535, "decay_scan: too many sequences");
  return f32 ? decay_scan_launch<float>(c, s) : decay_scan_launch<bf16>(c, s);
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

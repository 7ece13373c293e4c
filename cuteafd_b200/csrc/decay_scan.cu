// Linear attention with a decay per head or per key channel: retention and gated linear attention, which hyper-connected stacks run beside their
// attention, and HGRN2, a mixer of the mixed stacks.
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   out_t = norm(o_t) * silu(g_t)
// HGRN2 has no keys and no output gate: its forget gate f = l + (1 - l) sigmoid(z + b), with a learned lower bound l per channel, is the decay, and the
// key is what the gate gives up, 1 - f = (1 - l) sigmoid(-z - b); queries pass SiLU.
// Two forms.  Runs of up to DS_GROUP tokens (decoding, drafts, short portions; every run in the all-fp32 mode): one block per (head, sequence), the
// state crosses HBM once for the whole group.  Longer runs in chunks of DC_TOK tokens, all chunks of all heads in parallel:
//   chunk_states   D_c = sum_j decay(j -> end of chunk) k_j v_j^T          one tcgen05 product per (head, chunk), and the chunk's decays
//   chunk_scan     state in front of every chunk (operand tiles), state behind the run     elementwise over the chunks
//   chunk_out      o = (q k^T, decayed, causal) v + decay(start -> i) q S  three tcgen05 products per (head, chunk), output norm, gate
// Everything that is not a projection enters the products as two bf16 terms (value and rounding error, 16 bits of mantissa together), with fp32
// accumulators in tensor memory; the states stay fp32.  Per-channel decays are folded into q and k relative to the middle of the chunk, or of
// smaller blocks where they span too much for one reference (see `Channels`).
// (Sibling of linear_attn.cu, whose delta rule has no such form yet; the reference's linear-attention programs are AOT exports without sources.)
#define CA_PDL_CLASS 2
#include "stack_rows.cuh"
#include <climits>

// A state slot holds two states per head, each with the position it belongs to (-1: the zero state in front of a sequence).  A run starts from
// the state right in front of it and leaves its last state in the other place, so a repeated step repeats its writes.  Runs of up to `depth`
// tokens also leave their keys, decays and values (`ring`, by position): when some of them are taken back, the next run starts from the
// earlier state and absorbs the kept ones again.
#define DS_THREADS 256
#define DS_GROUP 16         // tokens of one pass over the state (at least 2 depth - 1)

template <typename T>
struct DecayScan {
  const T* q; const T* k; const T* v; const T* g; int ldp;  // column views of the projection rows: [H * dim], [H * dim], [H * vdim], [H * vdim]
  const float2* rope; int pairs;                            // [T, pairs], dimensions i and i + pairs turn together; null = none
  float q_scale, k_scale;
  const float* decay;                                       // [H] constant decays; null: alpha = sigmoid(a2 a1 + a2_b)^(1 / tau) per key channel
  const T* a1; const float* a2; const float* a2_b;          // [rank] columns of the projection rows, [H * dim, rank], [H * dim]
  int rank; float inv_tau;
  const float* forget_b; const float* lower;                // HGRN2 (null otherwise): bias and lower bound of the forget gate [H * dim], whose logits are k
  const float* norm; float eps, out_scale;                  // gain of the output norm [vdim], or null
  float* state; int* tags; float* ring;                     // [slots, 2, H, dim, vp], [slots, H, 2], [slots, depth, H, 2 dim + vp]
  const int* state_slot; const int* q_start; const int* q_len; const int* kv_len;
  T* out; int ldo;
  int H, dim, vdim, vp, depth, n_state;
  int long_from;                                            // runs of more tokens take the chunk kernels (bf16): only their replay is done here
  // scratch of the long form, a run's chunks consecutive from q_start / DC_TOK + sequence: contributions [chunks, H, dim, vp], factors
  // [chunks, H, 2 dim + 1] (decays of the chunk; what puts the state in front of it on the scale of the chunk's queries; how often the chunk is halved
  // for its scores), states as operand tiles [chunks, H, tile set]
  float* chunk_state; float* chunk_decay; uint8_t* chunk_tiles;
  int* status;
};

// HGRN2: (decay, key) of a channel from the forget gate's logit z (bias added) and lower bound l
__device__ __forceinline__ float2 forget_gate(float z, float l) {
  const float e = expf(-fabsf(z)), s = 1.f / (1.f + e), big = s, small = e * s;      // sigmoids of |z| and -|z|
  return make_float2(fmaf(1.f - l, z >= 0.f ? big : small, l), (1.f - l) * (z >= 0.f ? small : big));
}
__device__ __forceinline__ float silu_f(float z) { return __fdividef(z, 1.f + __expf(-fmaxf(z, -80.f))); }

// log alpha of a channel from its logit
__device__ __forceinline__ float log_decay(float z, float inv_tau) { return -(fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))) * inv_tau; }

struct ScanBase { int place, pos, replay; };               // where a run starts: which of the two states, its position, tokens to absorb again
__device__ __forceinline__ ScanBase scan_base(const int* tags, int p0) {
  if (p0 == 0) return ScanBase{0, -1, 0};
  const int c0 = tags[0] < p0 ? tags[0] : -2, c1 = tags[1] < p0 ? tags[1] : -2;
  const int pos = max(c0, c1);
  return ScanBase{c1 > c0 ? 1 : 0, pos, p0 - 1 - pos};
}

struct ScanTile {
  float* q; float* k; float* al; float* v; float* red; float* o;
  __device__ __forceinline__ ScanTile from(int t, int dim, int vp) const { return ScanTile{q + t * dim, k + t * dim, al + t * dim, v + t * vp, red, o}; }
};

// One pass over the state for `cnt` (<= NT) tokens of the tile, the first `replay` of which only advance it; partial outputs of this thread's
// rows stay in acc.
template <int NT>
__device__ __forceinline__ void scan_pass(const ScanTile& sm, const float* src, float* dst, float* mid, int cnt, int replay, int dim, int vp, int rg, int RG, int c4, float4 (&acc)[NT]) {
  constexpr int DS_ROWS = NT == 1 ? 8 : 4;                   // state rows a thread has in flight
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

// NT: tokens of a pass over the state.  One: decoding (several blocks per SM; kept rows of a drafted step are absorbed one by one in place).
template <typename T, int NT>
__global__ void __launch_bounds__(DS_THREADS, NT == 1 ? 3 : 1) decay_scan_kernel(const DecayScan<T> a, int cap) {
  pdl_launch(); pdl_wait();
  extern __shared__ float ds_smem[];
  __shared__ float red32[32];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, dim = a.dim, vp = a.vp;
  const int n = a.q_len[seq], p0 = a.kv_len[seq] - n, row0 = a.q_start[seq], slot = a.state_slot[seq];
  if (n <= 0) return;
  if (slot < 0 || slot >= a.n_state) { if (tid == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6F2); return; }
  ScanTile sm;
  sm.v = ds_smem; sm.red = sm.v + cap * vp; sm.o = sm.red + 4 * DS_THREADS;            // four at a time: multiples of 4 first
  sm.q = sm.o + vp; sm.k = sm.q + cap * dim; sm.al = sm.k + cap * dim;
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
  const bool only_replay = n > a.long_from;
  if (only_replay && !b.replay) return;

  for (int done = 0, first = 1; first || done < n; first = 0) {
    const int replay = first ? b.replay : 0, cnt = only_replay ? replay : min(cap, replay + n - done), fresh = cnt - replay;
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
      if (a.lower) {
        const float2 f = forget_gate(k + a.forget_b[h * dim + r], a.lower[h * dim + r]);
        al = f.x; k = f.y; q = q / (1.f + expf(-q));
      } else if (!a.decay) {
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
    if (only_replay) {                                      // the state moves up to the run's start, in its own place
      float4 acc[NT];
      if (works)
        for (int t = 0; t < cnt; t += NT) scan_pass<NT>(sm.from(t, dim, vp), t || b.pos >= 0 ? base : nullptr, base, nullptr, min(NT, cnt - t), 0, dim, vp, rg, RG, c4, acc);
      if (tid == 0) tags[b.place] = p0 - 1;
      return;
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
        const float g = a.g ? to_f(a.g[row * a.ldp + h * a.vdim + c]) : 0.f;
        a.out[row * a.ldo + h * a.vdim + c] = to_t<T>(sm.o[c] * inv * (a.norm ? a.norm[c] : 1.f) * (a.g ? g / (1.f + expf(-g)) : 1.f));
      }
    };
    float4 acc[NT];
    if constexpr (NT == 1) {
      for (int t = 0; t < cnt; ++t) {                       // a thread's part of the state is its own: no barrier between the passes
        const float* from = t == 0 ? src : (t <= replay ? base : last);
        if (works) scan_pass<1>(sm.from(t, dim, vp), from, t < replay ? base : last, nullptr, 1, 0, dim, vp, rg, RG, c4, acc);
        if (t >= replay) finish(t, acc[0]);
      }
    } else {
      if (works) scan_pass<NT>(sm, src, last, mid, cnt, replay, dim, vp, rg, RG, c4, acc);
#pragma unroll
      for (int t = 0; t < NT; ++t) if (t >= replay && t < cnt) finish(t, acc[t]);
    }
    done += fresh;
  }
  if (tid == 0) {
    tags[b.place] = b.replay ? p0 - 1 : b.pos;
    tags[1 - b.place] = p0 + n - 1;
  }
}

// ---------------------------------------------------------------- long runs in chunks
#define DC_TOK 128
#define DC_THREADS 512
#define DC_PARTS (DC_THREADS / 128)      // threads that share a row of an accumulator
#define DC_SPAN 80.f        // most binary digits that decays may span on either side of a common reference

// Operand tiles: 64 columns x 128 rows in 128-byte rows, 128-byte swizzle.  DB 64-wide blocks of key dimensions; value tiles have up to 4 blocks.
template <int DB>
struct ChunkSmem {
  static constexpr int TILE = 16384, HL = 2 * DB * TILE;               // an operand of key dimensions: values, then rounding errors
  static constexpr int SMALL = 4096;                                   // vectors, barrier, flags
  static constexpr int UNITS = 16 * DB * 64 * 4;                       // per-channel decays: sums over units of eight tokens
  static constexpr int X = 4 * TILE;                                   // decays [128, 64 DB] fp32, then the value tiles, then state tiles
  static constexpr int P = 4 * TILE;                                   // keys, then probabilities (two terms of two blocks), then state tiles
  static constexpr int STATES = HL + X + SMALL + UNITS, OUT = HL + P + X + SMALL + UNITS;
};

struct ChunkRun { int n, p0, row, len, ci, chunks; };                  // run, first row and length of the block's chunk, its place in the scratch
__device__ __forceinline__ bool chunk_of(const DecayScan<bf16>& a, int c, int seq, ChunkRun& r) {
  r.n = a.q_len[seq];
  r.chunks = (r.n + DC_TOK - 1) / DC_TOK;
  if (r.n <= a.long_from || c >= r.chunks) return false;
  const int row0 = a.q_start[seq];
  r.p0 = a.kv_len[seq] - r.n; r.row = row0 + c * DC_TOK; r.len = min(DC_TOK, r.n - c * DC_TOK); r.ci = row0 / DC_TOK + seq + c;
  return true;
}

__device__ __forceinline__ uint64_t dc_desc_mn(uint32_t saddr, uint32_t lbo) {      // MN-major, 128-byte swizzle: 64-wide blocks `lbo` bytes apart, 8-row groups 1024
  return (uint64_t)((saddr & 0x3FFFF) >> 4) | (uint64_t)(lbo >> 4) << 16 | (uint64_t)(1024 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)2 << 61;
}
__device__ __forceinline__ uint32_t dc_idesc(int n, int a_mn, int b_mn) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)a_mn << 15) | ((uint32_t)b_mn << 16) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
}
// Eight values at (row, column) of a tile set whose 64-wide blocks are `block` bytes apart.
__device__ __forceinline__ uint32_t tile_at(int row, int col, int block) { return (col >> 6) * block + row * 128 + ((((col >> 3) & 7) ^ (row & 7)) << 4); }
__device__ __forceinline__ void put8(uint8_t* tile, uint32_t at, const float* v) {
  uint32_t w[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) { const bf162 h = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]); w[j] = *(const uint32_t*)&h; }
  *(uint4*)(tile + at) = make_uint4(w[0], w[1], w[2], w[3]);
}
// A value and what bf16 rounds off it, `lo` bytes apart.
__device__ __forceinline__ void put8_two(uint8_t* tile, uint32_t at, int lo, const float* v) {
  float r[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) r[j] = v[j] - __bfloat162float(__float2bfloat16(v[j]));
  put8(tile, at, v);
  put8(tile + lo, at, r);
}

// Rows no kernel of the launch writes: loads may pass the stores in front of them.
__device__ __forceinline__ void ldg8(const bf16* p, float* v) {
  const uint4 q = __ldg((const uint4*)p);
  const bf162* h = (const bf162*)&q;
#pragma unroll
  for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(h[j]); v[2 * j] = f.x; v[2 * j + 1] = f.y; }
}
// Staged rows of float4: column groups of eight are turned by the row, so that a warp writes one column of 32 rows, or reads whole rows, without conflicts.
__device__ __forceinline__ int stage_col(int row, int c) { return c ^ (row & 7); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// Eight neighbouring dimensions of a head's projected row (zero past `dim`), rotated and scaled.  `vec`: rows and rotation allow 16-byte pieces.
__device__ __forceinline__ void head8(const bf16* row, int d0, int dim, const float2* cs, int pairs, float scale, bool vec, float* v) {
  if (d0 >= dim) {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = 0.f;
    return;
  }
  if (vec) {
    ldg8(row + d0, v);
    if (cs && d0 < 2 * pairs) {
      const bool lo = d0 < pairs;
      const int p0 = lo ? d0 : d0 - pairs;
      float u[8];
      ldg8(row + (lo ? d0 + pairs : p0), u);
#pragma unroll
      for (int j = 0; j < 8; j += 2) {                      // (cosine, sine) of two pairs
        const float4 c = __ldg((const float4*)(cs + p0 + j));
        v[j] = lo ? v[j] * c.x - u[j] * c.y : v[j] * c.x + u[j] * c.y;
        v[j + 1] = lo ? v[j + 1] * c.z - u[j + 1] * c.w : v[j + 1] * c.z + u[j + 1] * c.w;
      }
    }
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int d = d0 + j;
      v[j] = d < dim ? to_f(row[d]) : 0.f;
      if (cs && d < 2 * pairs) {
        const bool lo = d < pairs;
        const int pr = lo ? d : d - pairs;
        const float2 c = cs[pr];
        const float u = to_f(row[lo ? d + pairs : pr]);
        v[j] = lo ? v[j] * c.x - u * c.y : v[j] * c.x + u * c.y;
      }
    }
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) v[j] *= scale;
}

// How the chunk kernels get their decays: a constant per head, from a low-rank projection, from HGRN2's forget gate.
enum { DECAY_HEAD = 0, DECAY_LOW_RANK = 1, DECAY_FORGET = 2 };

// Per-channel decays: a thread owns two neighbouring channels of DC_SEG tokens - their decays, queries and keys stay in its registers, and every
// operand tile is written from there relative to whatever reference its product needs.  Sums of the decays' logarithms travel between the threads
// as sums over units of eight tokens.
//
// q_i k_j decays by 2^(P(i) - P(j)), P the running sum.  Referred to the middle of a block of D tokens, rows of its second half and keys of its first
// half have factors of at most one; rows and keys of the same half have, on either side of the middle, up to 2^(sum over D / 2 tokens).  So the
// chunk is cut into the largest blocks whose half-sums stay below DC_SPAN: their own scores are one product, and those between the halves of every
// larger block one more per halving (`depth` of them).  A chunk whose blocks of 16 exceed it (a channel that forgets at once) takes its scores
// from the ordinary cores, pair by pair.
#define DC_UNITS (DC_TOK / 8)
#define DC_PAIRWISE 4       // depth of such a chunk

// Decays below 2^-126 are zero.
__device__ __forceinline__ float exp2_f(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
// log2(1 - m) of a decay 1 - m, m up to 1/16: seven terms of the series, relative error below 2e-8.
__device__ __forceinline__ float log2_near_one(float m) {
  float p = fmaf(m, 1.f / 7.f, 1.f / 6.f);
  p = fmaf(m, p, 0.2f); p = fmaf(m, p, 0.25f); p = fmaf(m, p, 1.f / 3.f); p = fmaf(m, p, 0.5f); p = fmaf(m, p, 1.f);
  return m * p * -1.4426950408889634f;
}
// log2 of the sigmoid of z
__device__ __forceinline__ float log2_sigmoid(float z) {
  const float e = __expf(-fabsf(z)), far = -fmaf(fmaxf(-z, 0.f), 1.4426950408889634f, __log2f(1.f + e));
  return z > 2.75f ? log2_near_one(__fdividef(e, 1.f + e)) : far;
}

template <int DB, int MODE>
struct Channels {
  static constexpr int DP = DB * 64, PAIRS = DP / 2, SEGS = DC_THREADS / PAIRS, N = DC_TOK / SEGS;      // N: tokens of a thread
  float2 b[N];                                              // running sums of log2 decays
  uint32_t q[N], k[N];                                      // projected rows (bf16 pairs); FORGET: k are the gate's logits
  float2 bias, keep;                                        // FORGET: bias and 1 - lower bound
  int c, t0;                                                // first channel and token

  static __device__ __forceinline__ float2 wide(uint32_t v) { return __bfloat1622float2(*(const bf162*)&v); }

  // Two rows' worth of pairs.  No load stands behind a condition, so that all of them are in flight together.
  static __device__ __forceinline__ void pairs(const bf16* p, int ldp, int t0, int last, bool one, bool two, bool aligned, uint32_t (&v)[N]) {
    if (aligned) {
#pragma unroll
      for (int i = 0; i < N; ++i) v[i] = __ldg((const unsigned int*)(p + (size_t)min(t0 + i, last) * ldp));
    } else {
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const bf16* e = p + (size_t)min(t0 + i, last) * ldp;
        v[i] = __bfloat16_as_ushort(e[0]) | (uint32_t)__bfloat16_as_ushort(e[two ? 1 : 0]) << 16;
      }
    }
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] = !one || t0 + i > last ? 0u : (two ? v[i] : v[i] & 0xFFFFu);
  }
  __device__ __forceinline__ void load(const DecayScan<bf16>& a, int h, const ChunkRun& r, bool queries) {
    c = (threadIdx.x % PAIRS) * 2; t0 = (threadIdx.x / PAIRS) * N; len = r.len;
    const bool one = c < a.dim, two = c + 1 < a.dim, even = ((a.ldp | a.dim) & 1) == 0;
    const size_t at = (size_t)r.row * a.ldp + h * a.dim + (one ? c : 0);
    pairs(a.k + at, a.ldp, t0, len - 1, one, two, even && ((uintptr_t)a.k & 3) == 0, k);
    if (queries) pairs(a.q + at, a.ldp, t0, len - 1, one, two, even && ((uintptr_t)a.q & 3) == 0, q);
    if (MODE == DECAY_FORGET) {
      const float* fb = a.forget_b + h * a.dim + c;
      const float* lb = a.lower + h * a.dim + c;
      bias = make_float2(one ? fb[0] : 0.f, two ? fb[1] : 0.f);
      keep = make_float2(one ? 1.f - lb[0] : 0.f, two ? 1.f - lb[1] : 0.f);
    }
  }
  // Sigmoids of -x and -y at the price of one reciprocal.
  static __device__ __forceinline__ float2 sigmoid_neg2(float x, float y) {
    const float ex = 1.f + __expf(fminf(x, 40.f)), ey = 1.f + __expf(fminf(y, 40.f)), inv = __fdividef(1.f, ex * ey);
    return make_float2(inv * ey, inv * ex);
  }
  // log2(1 - m) of a decay 1 - m (what decays to less than 2^-26 in one step is gone)
  static __device__ __forceinline__ float gate_log(float m) {
    const float far = __log2f(fmaxf(1.f - m, 1.5e-8f));
    return m < 0.0625f ? log2_near_one(m) : far;
  }
  // FORGET: the key, (1 - l) sigmoid(-z).
  __device__ __forceinline__ float2 key(const DecayScan<bf16>& a, int i) const {
    const float2 v = wide(k[i]);
    if (MODE != DECAY_FORGET) return make_float2(v.x * a.k_scale, v.y * a.k_scale);
    const float2 s = sigmoid_neg2(v.x + bias.x, v.y + bias.y);
    return in_run(i) ? make_float2(keep.x * s.x, keep.y * s.y) : make_float2(0.f, 0.f);
  }
  __device__ __forceinline__ float2 query(const DecayScan<bf16>& a, int i) const {
    const float2 v = wide(q[i]);
    if (MODE != DECAY_FORGET) return make_float2(v.x * a.q_scale, v.y * a.q_scale);
    const float2 s = sigmoid_neg2(-v.x, -v.y);
    return make_float2(v.x * s.x, v.y * s.y);
  }
  int len;
  __device__ __forceinline__ bool in_run(int i) const { return t0 + i < len; }

  // Running sums; `X`: log2 decays [128, DP] (LOW_RANK); `units`: room for the units' sums [DC_UNITS, DP].  Ends with a barrier; all of `units` may be read.
  __device__ __forceinline__ void sums(const DecayScan<bf16>& a, const float* X, float* units) {
    float2 s = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < N; ++i) {
      float2 l;
      if (MODE == DECAY_FORGET) {
        const float2 m = key(a, i);
        l = make_float2(gate_log(m.x), gate_log(m.y));
      } else {
        l = *(const float2*)(X + (t0 + i) * DP + c);
      }
      if (i % 8 == 0) s = make_float2(0.f, 0.f);
      s.x += l.x; s.y += l.y;
      b[i] = s;
      if (i % 8 == 7) *(float2*)(units + ((t0 + i) >> 3) * DP + c) = s;
    }
    __syncthreads();
    float2 p = make_float2(0.f, 0.f);
    for (int u = 0; u < t0 / 8; ++u) { const float2 v = *(const float2*)(units + u * DP + c); p.x += v.x; p.y += v.y; }
#pragma unroll
    for (int i = 0; i < N; ++i) {
      if (i && i % 8 == 0) { const float2 v = *(const float2*)(units + ((t0 + i) / 8 - 1) * DP + c); p.x += v.x; p.y += v.y; }
      b[i].x += p.x; b[i].y += p.y;
    }
  }
  // Running sum in front of token `t` (a multiple of 8).
  __device__ __forceinline__ float2 front(const float* units, int t) const {
    float2 p = make_float2(0.f, 0.f);
    for (int u = 0; u < t / 8; ++u) { const float2 v = *(const float2*)(units + u * DP + c); p.x += v.x; p.y += v.y; }
    return p;
  }
  // Token i of this thread into a tile set, value and rounding error.
  __device__ __forceinline__ void put(uint8_t* tiles, int i, float2 v) const {
    const int t = t0 + i;
    const uint32_t at = tile_at(t, c & ~7, 16384) + (c & 7) * 2;
    const bf162 hi = __floats2bfloat162_rn(v.x, v.y);
    const float2 w = __bfloat1622float2(hi);
    const bf162 lo = __floats2bfloat162_rn(v.x - w.x, v.y - w.y);
    *(uint32_t*)(tiles + at) = *(const uint32_t*)&hi;
    *(uint32_t*)(tiles + at + DB * 16384) = *(const uint32_t*)&lo;
  }
};
// Smallest depth whose blocks' half-sums stay within DC_SPAN for this channel.
template <int DP>
__device__ __forceinline__ int span_depth(const float* units, int c) {
  float u[DC_UNITS];
#pragma unroll
  for (int j = 0; j < DC_UNITS; ++j) u[j] = units[j * DP + c];
  int depth = DC_PAIRWISE;
#pragma unroll
  for (int level = 3; level >= 0; --level) {                // halves of 8, 16, 32, 64 tokens: blocks of 16, 32, 64, 128
    const int n = 8 >> level;                               // units of a half
    float worst = 0.f;
#pragma unroll
    for (int j = 0; j < DC_UNITS; j += n) {
      float s = 0.f;
#pragma unroll
      for (int q = 0; q < n; ++q) s += u[j + q];
      worst = fminf(worst, s);
    }
    if (worst >= -DC_SPAN && depth == level + 1) depth = level;
  }
  return depth;
}

// log2 of the chunk's per-channel decays -> X [128, DP] (zero past the run's end and past `dim`); `stage`: 8 KB.
template <int DP>
__device__ __forceinline__ void chunk_logs(const DecayScan<bf16>& a, int h, const ChunkRun& r, float* X, float* stage) {
  const int tid = threadIdx.x, c = tid % DP;
  const float b = c < a.dim ? a.a2_b[h * a.dim + c] : 0.f;
  for (int r0 = 0; r0 < a.rank; r0 += 16) {
    __syncthreads();
    for (int i = tid; i < DC_TOK * 16; i += DC_THREADS) {
      const int t = i >> 4, q = r0 + (i & 15);
      const float v = to_f(a.a1[(size_t)(r.row + min(t, r.len - 1)) * a.ldp + min(q, a.rank - 1)]);
      stage[i] = t < r.len && q < a.rank ? v : 0.f;
    }
    float w[16];
#pragma unroll
    for (int q = 0; q < 16; ++q) w[q] = __ldg(a.a2 + (size_t)(h * a.dim + min(c, a.dim - 1)) * a.rank + min(r0 + q, a.rank - 1));
#pragma unroll
    for (int q = 0; q < 16; ++q) w[q] = c < a.dim && r0 + q < a.rank ? w[q] : 0.f;
    __syncthreads();
    for (int t = tid / DP; t < DC_TOK; t += DC_THREADS / DP) {
      float z = r0 ? X[t * DP + c] : b;
#pragma unroll
      for (int q = 0; q < 16; q += 4) {
        const float4 s = *(const float4*)(stage + t * 16 + q);
        z = fmaf(w[q], s.x, z); z = fmaf(w[q + 1], s.y, z); z = fmaf(w[q + 2], s.z, z); z = fmaf(w[q + 3], s.w, z);
      }
      X[t * DP + c] = r0 + 16 < a.rank ? z : (t < r.len && c < a.dim ? log2_sigmoid(z) * a.inv_tau : 0.f);
    }
  }
  __syncthreads();
}

__device__ __forceinline__ void load_values(const DecayScan<bf16>& a, int h, const ChunkRun& r, uint8_t* sV, int VB) {
  const bool vec = ((a.vdim | a.ldp) & 7) == 0 && ((uintptr_t)a.v & 15) == 0;
  for (int i = threadIdx.x; i < DC_TOK * VB * 8; i += DC_THREADS) {
    const int t = i / (VB * 8), c0 = (i % (VB * 8)) * 8;
    const bool in = t < r.len && c0 < a.vdim;
    const bf16* src = a.v + (size_t)(r.row + t) * a.ldp + h * a.vdim + c0;
    uint8_t* dst = sV + tile_at(t, c0, 16384);
    if (in && vec) { cp_async16(dst, src); continue; }      // (the caller waits for the copies)
    float e[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) e[j] = in && c0 + j < a.vdim ? to_f(src[j]) : 0.f;
    put8(dst, 0, e);
  }
}

__device__ __forceinline__ float decay_log2(float d) { return fmaxf(log2f(d), -1e30f); }      // (a decay of zero forgets everything but the token itself)

// Barrier, tensor memory and the end of a chunk block.
struct ChunkSync {
  uint64_t* bar; int* abortp; uint32_t tmem; int ph; int* status;
  // All threads: wait for the products committed last.
  __device__ __forceinline__ void wait(int where) {
    if (!mbar_wait_bounded(bar, ph, (volatile int*)abortp)) ca_dev_fail(status, CA_DEV_TIMEOUT_EPILOGUE, where);
    ph ^= 1;
    tc_fence_after();
  }
  __device__ __forceinline__ void publish() { fence_proxy_async_smem(); tc_fence_before(); __syncthreads(); tc_fence_after(); }
};
__device__ __forceinline__ ChunkSync chunk_begin(uint8_t* small, int cols, int* status) {
  uint64_t* bar = (uint64_t*)small;
  uint32_t* slot = (uint32_t*)(small + 8);
  int* abortp = (int*)(small + 16);
  if (threadIdx.x == 0) { mbar_init(bar, 1); *abortp = 0; fence_barrier_init(); }
  if (threadIdx.x >> 5 == 1) { tmem_alloc(slot, cols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  return ChunkSync{bar, abortp, *slot, 0, status};
}
__device__ __forceinline__ void chunk_end(const ChunkSync& y, int cols) {
  if (*(volatile int*)y.abortp && threadIdx.x < 32) { const uint64_t t0 = globaltimer_ns(); while (globaltimer_ns() - t0 < 200000) __nanosleep(1000); }
  tc_fence_before();
  __syncthreads();
  if (threadIdx.x >> 5 == 1) tmem_dealloc(y.tmem, cols);
}

// D_c = sum_j decay(j -> end) k_j v_j^T of one head and chunk, rows of key dimensions; the decays of the whole chunk.
template <int DB, int MODE>
__global__ void __launch_bounds__(DC_THREADS, 1) chunk_states_kernel(const __grid_constant__ DecayScan<bf16> a) {
  pdl_launch(); pdl_wait();
  using Sm = ChunkSmem<DB>;
  constexpr int DP = DB * 64;
  extern __shared__ __align__(1024) uint8_t dc_smem[];
  const int h = blockIdx.x, tid = threadIdx.x;
  ChunkRun r;
  if (!chunk_of(a, blockIdx.y, blockIdx.z, r)) return;                // block-uniform
  if (smem_u32(dc_smem) & 1023) { if (tid == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6F4); return; }
  uint8_t* sK = dc_smem; uint8_t* sX = sK + Sm::HL; uint8_t* small = sX + Sm::X;
  ChunkSync y = chunk_begin(small, 256, a.status);
  const int VB = (a.vp + 63) / 64;
  float* factors = a.chunk_decay + ((size_t)r.ci * a.H + h) * (2 * a.dim + 1);
  if constexpr (MODE != DECAY_HEAD) {
    float* units = (float*)(small + Sm::SMALL);
    Channels<DB, MODE> ch;
    ch.load(a, h, r, false);
    if (MODE == DECAY_FORGET) load_values(a, h, r, sX, VB);
    else chunk_logs<DP>(a, h, r, (float*)sX, (float*)sK);
    ch.sums(a, (const float*)sX, units);
    if (MODE != DECAY_FORGET) load_values(a, h, r, sX, VB);           // (every thread has read its decays)
    int* depth = (int*)(small + 24);
    if (tid == 0) *depth = 0;
    const float2 total = ch.front(units, DC_TOK);
    __syncthreads();
    float first = 0.f, all = 0.f;
    if (tid < DP) {
      const int d = span_depth<DP>(units, tid);
      if (d) atomicMax(depth, d);
      for (int u = 0; u < DC_UNITS; ++u) { all += units[u * DP + tid]; if (u == DC_UNITS / 2 - 1) first = all; }
    }
    __syncthreads();
    if (tid == 0) factors[2 * a.dim] = (float)*depth;
    if (tid < a.dim) { factors[tid] = exp2f(all); factors[a.dim + tid] = *depth ? 1.f : exp2f(first); }
#pragma unroll
    for (int i = 0; i < Channels<DB, MODE>::N; ++i) {
      const float2 k = ch.key(a, i);
      ch.put(sK, i, make_float2(k.x * exp2_f(total.x - ch.b[i].x), k.y * exp2_f(total.y - ch.b[i].y)));
    }
  } else {
    const bool vec = ((a.dim | a.ldp | (a.rope ? a.pairs : 0)) & 7) == 0 && ((uintptr_t)a.k & 15) == 0;
    const float l2 = decay_log2(a.decay[h]);
    load_values(a, h, r, sX, VB);
    if (tid < a.dim) { factors[tid] = exp2f(l2 * (float)r.len); factors[a.dim + tid] = 1.f; }
#pragma unroll 4
    for (int i = tid; i < DC_TOK * DB * 8; i += DC_THREADS) {
      const int t = i / (DB * 8), d0 = (i % (DB * 8)) * 8;
      float v[8];
      if (t < r.len) {
        const size_t row = r.row + t;
        head8(a.k + row * a.ldp + h * a.dim, d0, a.dim, a.rope ? a.rope + row * a.pairs : nullptr, a.pairs, a.k_scale, vec, v);
        const float f = exp2f(l2 * (float)(r.len - 1 - t));
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] *= f;
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = 0.f;
      }
      put8_two(sK, tile_at(t, d0, Sm::TILE), DB * Sm::TILE, v);
    }
  }
  cp_async_wait();
  y.publish();
  if (tid == 0) {
    const uint32_t id = dc_idesc(VB * 64, 1, 1);
    for (int part = 0; part < 2; ++part)
      for (int k = 0; k < DC_TOK / 16; ++k)
        tc_mma_f16(y.tmem, dc_desc_mn(smem_u32(sK) + part * DB * Sm::TILE + k * 2048, Sm::TILE), dc_desc_mn(smem_u32(sX) + k * 2048, Sm::TILE), id, (part | k) ? 1u : 0u);
    tc_commit(y.bar);
  }
  __syncwarp();
  y.wait(0x6F5);
  const int warp = tid >> 5, row = (warp & 3) * 32 + (tid & 31), pitch = VB * 16;
  constexpr int PW = 64 / DC_PARTS;                                   // columns of a 64-wide block that a thread takes
  float4* stage = (float4*)sK;                                        // (keys and values have been read: rows of key dimensions, whole lines to memory)
  for (int c = (warp >> 2) * VB * PW; c < ((warp >> 2) + 1) * VB * PW; c += 16) {
    uint32_t o[16];
    tmem_ld_x16(y.tmem + ((uint32_t)((warp & 3) * 32) << 16) + c, o);
    tc_wait_ld();
    if (row < DP)
#pragma unroll
      for (int j = 0; j < 4; ++j) stage[row * pitch + stage_col(row, c / 4 + j)] = *(const float4*)(o + 4 * j);
  }
  __syncthreads();
  float4* dst = (float4*)(a.chunk_state + ((size_t)r.ci * a.H + h) * a.dim * a.vp);
  for (int i = tid; i < a.dim * (a.vp / 4); i += DC_THREADS) {
    const int d = i / (a.vp / 4), c = i % (a.vp / 4);
    dst[i] = stage[d * pitch + stage_col(d, c)];
  }
  chunk_end(y, 256);
}

// The chunks' contributions become the states in front of the chunks, as the operand tiles (values, then rounding errors) of the output kernel; the
// state behind the run goes to the slot.
template <int DB>
__global__ void __launch_bounds__(128) chunk_scan_kernel(const DecayScan<bf16> a) {
  pdl_launch(); pdl_wait();
  const int h = blockIdx.y, seq = blockIdx.z, e = (blockIdx.x * 128 + threadIdx.x) * 4, one = a.dim * a.vp;
  ChunkRun r;
  if (!chunk_of(a, 0, seq, r) || e >= one) return;
  const int slot = a.state_slot[seq];
  if (slot < 0 || slot >= a.n_state) { if (e == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6F2); return; }
  const ScanBase b = scan_base(a.tags + ((size_t)slot * a.H + h) * 2, r.p0);
  if (b.pos < -1 || b.replay) { if (e == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6F3); return; }
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (b.pos >= 0) S = *(const float4*)(a.state + (((size_t)slot * 2 + b.place) * a.H + h) * one + e);
  const int row = e / a.vp, col = e % a.vp, half = (a.vp + 63) / 64 * DB * 64 * 128;
  const float* D = a.chunk_state + ((size_t)r.ci * a.H + h) * one + e;
  const float* dec = a.chunk_decay + ((size_t)r.ci * a.H + h) * (2 * a.dim + 1) + row;
  uint8_t* tile = a.chunk_tiles + ((size_t)r.ci * a.H + h) * 2 * half + tile_at(row, col, DB * 64 * 128) + (col & 7) * 2;
  const size_t step = (size_t)a.H * one, dstep = (size_t)a.H * (2 * a.dim + 1), tstep = (size_t)a.H * 2 * half;
  for (int c0 = 0; c0 < r.chunks; c0 += 8) {
    float4 d[8]; float f[8], m[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = min(c0 + j, r.chunks - 1);
      d[j] = __ldg((const float4*)(D + c * step)); f[j] = __ldg(dec + c * dstep); m[j] = __ldg(dec + c * dstep + a.dim);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c0 + j >= r.chunks) break;
      const float v[4] = {S.x * m[j], S.y * m[j], S.z * m[j], S.w * m[j]};
      float lo[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) lo[q] = v[q] - __bfloat162float(__float2bfloat16(v[q]));
      store4<bf16>((bf16*)(tile + (c0 + j) * tstep), v);
      store4<bf16>((bf16*)(tile + (c0 + j) * tstep + half), lo);
      S.x = fmaf(f[j], S.x, d[j].x); S.y = fmaf(f[j], S.y, d[j].y); S.z = fmaf(f[j], S.z, d[j].z); S.w = fmaf(f[j], S.w, d[j].w);
    }
  }
  *(float4*)(a.state + (((size_t)slot * 2 + 1 - b.place) * a.H + h) * one + e) = S;
}

template <int DB, int MODE>
__global__ void __launch_bounds__(DC_THREADS, 1) chunk_out_kernel(const __grid_constant__ DecayScan<bf16> a) {
  pdl_launch(); pdl_wait();
  using Sm = ChunkSmem<DB>;
  constexpr int DP = DB * 64, T = Sm::TILE;
  extern __shared__ __align__(1024) uint8_t dc_smem[];
  const int h = blockIdx.x, seq = blockIdx.z, tid = threadIdx.x;
  ChunkRun r;
  if (!chunk_of(a, blockIdx.y, seq, r)) return;                       // block-uniform
  const int slot = a.state_slot[seq];
  if (slot < 0 || slot >= a.n_state || (smem_u32(dc_smem) & 1023)) { if (tid == 0) ca_dev_fail(a.status, CA_DEV_BAD_INDEX, 0x6F6); return; }
  uint8_t* sQ = dc_smem; uint8_t* sP = sQ + Sm::HL; uint8_t* sX = sP + Sm::P; uint8_t* small = sX + Sm::X;
  float* ssum = (float*)(small + 64);                                 // [DC_PARTS, 128]
  float* gain = ssum + DC_PARTS * 128;                                // [256]
  uint64_t* tiles_bar = (uint64_t*)(small + 32);                      // [2]
  if (tid == 0) { mbar_init(tiles_bar, 1); mbar_init(tiles_bar + 1, 1); }
  if (a.norm && tid < a.vdim) gain[tid] = a.norm[tid];
  ChunkSync y = chunk_begin(small, 512, a.status);
  const uint32_t O1 = 0, O2 = 256, SC = 256;                          // scores stand where the state's share is accumulated later
  constexpr int KW = DC_TOK / DC_PARTS, PW = 64 / DC_PARTS;             // keys, and columns of a 64-wide block of values, that a thread takes of its row
  const int VB = (a.vp + 63) / 64, warp = tid >> 5, part = warp >> 2, row = (warp & 3) * 32 + (tid & 31);
  const uint32_t lanes = (uint32_t)((warp & 3) * 32) << 16;
  const uint32_t q0 = smem_u32(sQ), k0 = smem_u32(sP);
  auto score = [&](uint32_t col) {                                    // one thread: queries x keys, value x value, value x error, error x value
    const uint32_t id = dc_idesc(DC_TOK, 0, 0);
    for (int part = 0; part < 3; ++part) {
      const uint32_t qa = q0 + (part == 2 ? DB * T : 0), kb = k0 + (part == 1 ? DB * T : 0);
      for (int b = 0; b < DB; ++b)
        for (int k = 0; k < 4; ++k) tc_mma_f16(y.tmem + col, umma_desc_sw128(qa + b * T) + 2 * k, umma_desc_sw128(kb + b * T) + 2 * k, id, (part | b | k) ? 1u : 0u);
    }
    tc_commit(y.bar);
  };
  float sc[KW];                                                       // this thread's scores: its row, keys [part * KW, + KW)
  float l2 = 0.f;
  if constexpr (MODE != DECAY_HEAD) {
    using Ch = Channels<DB, MODE>;
    float* X = (float*)sX;
    float* units = (float*)(small + Sm::SMALL);
    const int depth = (int)a.chunk_decay[((size_t)r.ci * a.H + h) * (2 * a.dim + 1) + 2 * a.dim];
    Ch ch;
    ch.load(a, h, r, true);
    if (MODE == DECAY_FORGET) { if (depth < DC_PAIRWISE) load_values(a, h, r, sX, VB); }
    else chunk_logs<DP>(a, h, r, X, (float*)sQ);
    ch.sums(a, X, units);
    if (depth < DC_PAIRWISE) {
      if (MODE != DECAY_FORGET) load_values(a, h, r, sX, VB);         // (every thread has read its decays)
#pragma unroll 1
      for (int l = 0; l <= depth; ++l) {                              // blocks of 128 >> l tokens, referred to the running sums in front of their middles
        const int half = DC_TOK >> (l + 1);
        const float2 ref = ch.front(units, (ch.t0 & -(2 * half)) + half);
#pragma unroll
        for (int i = 0; i < Ch::N; ++i) {
          // rows that have no part in this product hold zeros
          const bool second = (ch.t0 + i) & half, as_q = l == depth || second, as_k = l == depth || !second;
          const float2 x = make_float2(ch.b[i].x - ref.x, ch.b[i].y - ref.y), q = ch.query(a, i), k = ch.key(a, i);
          ch.put(sQ, i, as_q ? make_float2(q.x * exp2_f(x.x), q.y * exp2_f(x.y)) : make_float2(0.f, 0.f));
          ch.put(sP, i, as_k ? make_float2(k.x * exp2_f(-x.x), k.y * exp2_f(-x.y)) : make_float2(0.f, 0.f));
        }
        y.publish();
        if (tid == 0) score((SC + l * 128) & 511);
        __syncwarp();
        y.wait(0x6F7);
      }
#pragma unroll
      for (int c = 0; c < KW; c += 16) {
#pragma unroll
        for (int j = 0; j < 16; ++j) sc[c + j] = 0.f;
#pragma unroll 1
        for (int l = 0; l <= depth; ++l) {
          uint32_t o[16];
          tmem_ld_x16(y.tmem + lanes + ((SC + l * 128) & 511) + part * KW + c, o);
          tc_wait_ld();
          const int half = DC_TOK >> (l + 1);
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const int key = part * KW + c + j;
            const bool same = ((row ^ key) & -(2 * half)) == 0;
            if (same && key <= row && (l == depth || ((row & half) && !(key & half)))) sc[c + j] = __uint_as_float(o[j]);
          }
        }
      }
    } else {
      // pair by pair: the decays between two tokens as the difference of their sums
      __syncthreads();                                                // the units' sums (LOW_RANK: the logarithms) have been read
#pragma unroll
      for (int i = 0; i < Ch::N; ++i) { *(float2*)(X + (ch.t0 + i) * DP + ch.c) = ch.b[i]; ch.put(sP, i, ch.key(a, i)); ch.put(sQ, i, ch.query(a, i)); }
      __syncthreads();
#pragma unroll
      for (int j = 0; j < KW; ++j) sc[j] = 0.f;
      if (part * KW <= (warp & 3) * 32 + 31)                          // warp-uniform: some key is not behind every row of the warp
        for (int d0 = 0; d0 < a.dim; d0 += 8) {
          float q[8], e[8], x[8];
          const uint8_t* qt = sQ + tile_at(row, d0, T);
          load8<bf16>((const bf16*)qt, q);
          load8<bf16>((const bf16*)(qt + DB * T), e);
#pragma unroll
          for (int j = 0; j < 8; ++j) { q[j] += e[j]; x[j] = X[row * DP + d0 + j]; }
#pragma unroll
          for (int j = 0; j < KW; ++j) {
            const int key = part * KW + j;
            const uint8_t* at = sP + tile_at(key, d0, T);
            float k[8], lo[8];
            load8<bf16>((const bf16*)at, k);
            load8<bf16>((const bf16*)(at + DB * T), lo);
#pragma unroll
            for (int e2 = 0; e2 < 8; ++e2) sc[j] = fmaf(q[e2] * (k[e2] + lo[e2]), exp2f(x[e2] - X[key * DP + d0 + e2]), sc[j]);
          }
        }
#pragma unroll
      for (int j = 0; j < KW; ++j) if (part * KW + j > row || row >= r.len) sc[j] = 0.f;       // (may not be a number)
      __syncthreads();                                                // the decays have been read
      load_values(a, h, r, sX, VB);
    }
    if (depth)                                                        // the state is decayed from the chunk's start
#pragma unroll
      for (int i = 0; i < Ch::N; ++i) { const float2 q = ch.query(a, i); ch.put(sQ, i, make_float2(q.x * exp2_f(ch.b[i].x), q.y * exp2_f(ch.b[i].y))); }
  } else {
    const bool vec = ((a.dim | a.ldp | (a.rope ? a.pairs : 0)) & 7) == 0 && (((uintptr_t)a.q | (uintptr_t)a.k) & 15) == 0;
    l2 = decay_log2(a.decay[h]);
    load_values(a, h, r, sX, VB);
#pragma unroll 2
    for (int i = tid; i < DC_TOK * DB * 8; i += DC_THREADS) {
      const int t = i / (DB * 8), d0 = (i % (DB * 8)) * 8;
      float q[8], k[8];
      if (t < r.len) {
        const size_t gr = r.row + t;
        const float2* cs = a.rope ? a.rope + gr * a.pairs : nullptr;
        head8(a.q + gr * a.ldp + h * a.dim, d0, a.dim, cs, a.pairs, a.q_scale, vec, q);
        head8(a.k + gr * a.ldp + h * a.dim, d0, a.dim, cs, a.pairs, a.k_scale, vec, k);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) q[j] = k[j] = 0.f;
      }
      put8_two(sQ, tile_at(t, d0, T), DB * T, q);
      put8_two(sP, tile_at(t, d0, T), DB * T, k);
    }
    y.publish();
    if (tid == 0) score(SC);
    __syncwarp();
    y.wait(0x6F7);
#pragma unroll
    for (int c = 0; c < KW; c += 16) {
      uint32_t o[16];
      tmem_ld_x16(y.tmem + lanes + SC + part * KW + c, o);
      tc_wait_ld();
#pragma unroll
      for (int j = 0; j < 16; ++j) {
        const int back = row - (part * KW + c + j);
        sc[c + j] = back < 0 ? 0.f : __uint_as_float(o[j]) * exp2f(l2 * (float)back);
      }
    }
  }
  tc_fence_before();
  __syncthreads();                                                    // keys and scores have been read
  tc_fence_after();
#pragma unroll
  for (int c = 0; c < KW; c += 8) put8_two(sP, tile_at(row, part * KW + c, T), 2 * T, sc + c);
  cp_async_wait();
  y.publish();
  if (tid == 0) {
    const uint32_t id = dc_idesc(VB * 64, 0, 1), p0 = smem_u32(sP), v0 = smem_u32(sX);
    for (int part = 0; part < 2; ++part)
      for (int k = 0; k < DC_TOK / 16; ++k)
        tc_mma_f16(y.tmem + O1, umma_desc_sw128(p0 + part * 2 * T + (k >> 2) * T) + 2 * (k & 3), dc_desc_mn(v0 + k * 2048, T), id, (part | k) ? 1u : 0u);
    tc_commit(y.bar);
  }
  __syncwarp();
  y.wait(0x6F8);
  // the state in front of the chunk takes the place of probabilities and values; its rounding errors arrive under the first two products
  if (tid == 0) {
    const uint32_t bytes = VB * DP * 128;
    const uint8_t* S = a.chunk_tiles + ((size_t)r.ci * a.H + h) * 2 * bytes;
    for (int part = 0; part < 2; ++part) {
      mbar_expect_tx(tiles_bar + part, bytes);
      bulk_load_1d(part ? sX : sP, S + part * bytes, bytes, tiles_bar + part);
    }
    const uint32_t id = dc_idesc(VB * 64, 0, 1);
    for (int part = 0; part < 3; ++part) {                            // value x value, error x value, value x error
      if (part != 1 && !mbar_wait_bounded(tiles_bar + part / 2, 0, (volatile int*)y.abortp)) ca_dev_fail(a.status, CA_DEV_TIMEOUT_PRODUCER, 0x6FA);
      const uint32_t qa = q0 + (part == 1 ? DB * T : 0), sb = smem_u32(part == 2 ? sX : sP);
      for (int k = 0; k < DP / 16; ++k) tc_mma_f16(y.tmem + O2, umma_desc_sw128(qa + (k >> 2) * T) + 2 * (k & 3), dc_desc_mn(sb + k * 2048, DP * 128), id, (part | k) ? 1u : 0u);
    }
    tc_commit(y.bar);
  }
  __syncwarp();
  // the gates arrive under these products, in the order of the stores: piece i of a thread is eight columns of a row
  const int c_lo = part * VB * PW, c_hi = c_lo + VB * PW;
  const bool vout = ((a.vdim | a.ldp | a.ldo) & 7) == 0 && (((uintptr_t)a.g | (uintptr_t)a.out) & 15) == 0;
  constexpr int NG = DC_TOK * 32 / DC_THREADS;
  uint4 gates[NG];
  if (a.g && vout) {
#pragma unroll
    for (int p = 0; p < NG; ++p) {
      const int t = min((tid + p * DC_THREADS) >> 5, r.len - 1), c = min((tid & 31) * 8, a.vdim - 8);
      gates[p] = __ldg((const uint4*)(a.g + (size_t)(r.row + t) * a.ldp + h * a.vdim + c));
    }
  }
  y.wait(0x6F9);
  // sum of both shares; its norm; rows through shared memory (nothing else is read there any more), gated and stored in whole lines
  const float f2 = MODE != DECAY_HEAD ? 1.f : exp2f(l2 * (float)(row + 1));
  float4* stage = (float4*)sP;
  const int pitch = VB * 16;
  float ss = 0.f;
  for (int c = c_lo; c < c_hi; c += 16) {
    uint32_t o[16], s[16];
    tmem_ld_x16(y.tmem + lanes + O1 + c, o);
    tmem_ld_x16(y.tmem + lanes + O2 + c, s);
    tc_wait_ld();
#pragma unroll
    for (int j = 0; j < 16; j += 4) {
      float4 v;
      v.x = fmaf(f2, __uint_as_float(s[j]), __uint_as_float(o[j])); v.y = fmaf(f2, __uint_as_float(s[j + 1]), __uint_as_float(o[j + 1]));
      v.z = fmaf(f2, __uint_as_float(s[j + 2]), __uint_as_float(o[j + 2])); v.w = fmaf(f2, __uint_as_float(s[j + 3]), __uint_as_float(o[j + 3]));
      ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);        // columns past vdim are zero
      stage[row * pitch + stage_col(row, (c + j) / 4)] = v;
    }
  }
  ssum[part * 128 + row] = ss;
  __syncthreads();
  // a thread has the same columns of NG rows
  const int c = (tid & 31) * 8;
  float gains[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) gains[j] = a.out_scale * (a.norm ? gain[min(c + j, a.vdim - 1)] : 1.f);
#pragma unroll
  for (int p = 0; p < NG; ++p) {
    const int t = (tid + p * DC_THREADS) >> 5;
    if (t >= r.len || c >= a.vdim) break;
    const float4 u = stage[t * pitch + stage_col(t, c / 4)], w = stage[t * pitch + stage_col(t, c / 4 + 1)];
    float v[8] = {u.x, u.y, u.z, u.w, w.x, w.y, w.z, w.w}, s = 0.f;
#pragma unroll
    for (int q = 0; q < DC_PARTS; ++q) s += ssum[q * 128 + t];
    const float inv = rsqrtf(s / (float)a.vdim + a.eps);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] *= inv * gains[j];
    bf16* dst = a.out + (size_t)(r.row + t) * a.ldo + h * a.vdim + c;
    if (vout) {
      if (a.g) {
        const bf162* gp = (const bf162*)&gates[p];
#pragma unroll
        for (int j = 0; j < 4; ++j) { const float2 g = __bfloat1622float2(gp[j]); v[2 * j] *= silu_f(g.x); v[2 * j + 1] *= silu_f(g.y); }
      }
      store8<bf16>(dst, v);
    } else {
      const bf16* g = a.g ? a.g + (size_t)(r.row + t) * a.ldp + h * a.vdim + c : nullptr;
#pragma unroll
      for (int j = 0; j < 8; ++j) if (c + j < a.vdim) dst[j] = __float2bfloat16(g ? v[j] * silu_f(to_f(g[j])) : v[j]);
    }
  }
  if (tid == 0 && (int)blockIdx.y == r.chunks - 1) {                  // no other block of this launch reads the tags
    int* tags = a.tags + ((size_t)slot * a.H + h) * 2;
    const ScanBase b = scan_base(tags, r.p0);
    tags[b.place] = b.pos; tags[1 - b.place] = r.p0 + r.n - 1;
  }
  chunk_end(y, 512);
}

// ---------------------------------------------------------------- C ABI
struct CaDecayScan {
  const void* q; const void* k; const void* v; const void* g; const void* rope; const float* decay; const void* a1; const float* a2; const float* a2_b; const float* norm;
  float* state; int* tags; float* ring; const int* state_slot; const int* q_start; const int* q_len; const int* kv_len; void* out; float* chunk_state; float* chunk_decay; void* chunk_tiles; int* status; const float* forget_b; const float* lower;
  int ldp, pairs, rank, ldo, H, dim, vdim, vp, depth, n_state, n_seq, max_q_len, T, chunks; float q_scale, k_scale, inv_tau, eps, out_scale;
};

template <typename T>
static DecayScan<T> decay_scan_args(const CaDecayScan* c, bool chunked) {
  return DecayScan<T>{(const T*)c->q, (const T*)c->k, (const T*)c->v, (const T*)c->g, c->ldp, (const float2*)c->rope, c->pairs, c->q_scale, c->k_scale, c->decay, (const T*)c->a1, c->a2,
                      c->a2_b, c->rank, c->inv_tau, c->forget_b, c->lower, c->norm, c->eps, c->out_scale, c->state, c->tags, c->ring, c->state_slot, c->q_start, c->q_len, c->kv_len, (T*)c->out, c->ldo,
                      c->H, c->dim, c->vdim, c->vp, c->depth, c->n_state, chunked ? DS_GROUP : INT_MAX, c->chunk_state, c->chunk_decay, (uint8_t*)c->chunk_tiles, c->status};
}

template <typename K>
static int dynamic_smem(K kern, int bytes, bool (&done)[64]) {
  int dev = 0; cudaGetDevice(&dev);
  if (!done[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e != cudaSuccess) return ca_cuda(e, "cudaFuncSetAttribute(decay_scan)");
    done[dev & 63] = true;
  }
  return CA_OK;
}

template <typename T, int NT>
static int decay_scan_launch(const CaDecayScan* c, bool chunked, cudaStream_t s) {
  const int longest = chunked ? DS_GROUP : c->max_q_len;
  const int cap = longest + c->depth - 1 < DS_GROUP ? longest + c->depth - 1 : DS_GROUP;
  const size_t smem = ((size_t)cap * (3 * c->dim + c->vp) + 4 * DS_THREADS + c->vp) * sizeof(float);
  static bool attr_set[64] = {false};
  const int rc = dynamic_smem(decay_scan_kernel<T, NT>, 200 * 1024, attr_set);
  if (rc) return rc;
  CA_REQUIRE(smem <= 200 * 1024, "decay_scan: heads of %d x %d do not fit shared memory", c->dim, c->vdim);
  CA_LAUNCH_PDL((decay_scan_kernel<T, NT>), dim3(c->H, c->n_seq), DS_THREADS, smem, s, decay_scan_args<T>(c, chunked), cap);
  CA_CHECK_LAUNCH("decay_scan");
  return CA_OK;
}

template <int DB, int MODE>
static int chunk_launch(const CaDecayScan* c, cudaStream_t s) {
  const DecayScan<bf16> a = decay_scan_args<bf16>(c, true);
  const int chunks = (c->max_q_len + DC_TOK - 1) / DC_TOK;
  const dim3 grid(c->H, chunks, c->n_seq);
  static bool states_set[64] = {false}, out_set[64] = {false};
  int rc = dynamic_smem(chunk_states_kernel<DB, MODE>, ChunkSmem<DB>::STATES, states_set);
  if (!rc) rc = dynamic_smem(chunk_out_kernel<DB, MODE>, ChunkSmem<DB>::OUT, out_set);
  if (rc) return rc;
  CA_LAUNCH_PDL((chunk_states_kernel<DB, MODE>), grid, DC_THREADS, ChunkSmem<DB>::STATES, s, a);
  CA_CHECK_LAUNCH("decay_scan chunk states");
  CA_LAUNCH_PDL((chunk_scan_kernel<DB>), dim3((c->dim * c->vp / 4 + 127) / 128, c->H, c->n_seq), 128, 0, s, a);
  CA_CHECK_LAUNCH("decay_scan chunk scan");
  CA_LAUNCH_PDL((chunk_out_kernel<DB, MODE>), grid, DC_THREADS, ChunkSmem<DB>::OUT, s, a);
  CA_CHECK_LAUNCH("decay_scan chunk outputs");
  return CA_OK;
}

// Whether the chunk kernels take a step's long runs.
static bool chunkable(const CaDecayScan* c, int f32) { return !f32 && c->chunk_state && c->chunk_decay && c->chunk_tiles && c->dim <= 128 && c->vdim <= 256 && c->max_q_len > DS_GROUP && (c->decay || !c->pairs); }

extern "C" int cuteafd_decay_scan(const CaDecayScan* c, int f32, cudaStream_t s) {
  CA_REQUIRE(c && c->q && c->k && c->v && (c->g || c->lower) && c->state && c->tags && c->ring && c->state_slot && c->q_start && c->q_len && c->kv_len && c->out, "decay_scan: null argument");
  CA_REQUIRE(!c->lower || (c->forget_b && !c->decay && !c->a1 && c->pairs == 0), "decay_scan: a forget gate has a bias, and no other decays or rotation");
  CA_REQUIRE(c->lower || c->decay || (c->a1 && c->a2 && c->a2_b && c->rank >= 1), "decay_scan: neither constant decays nor a projection of them");
  CA_REQUIRE(c->H >= 1 && c->dim >= 1 && c->dim <= 512 && c->vdim >= 1 && c->vp % 4 == 0 && c->vp >= c->vdim && c->vp <= 4 * DS_THREADS, "decay_scan: heads of %d x %d (at most 512 x %d)", c->dim, c->vdim, 4 * DS_THREADS);
  CA_REQUIRE(c->pairs >= 0 && 2 * c->pairs <= c->dim && (c->pairs == 0 || c->rope) && c->depth >= 1 && 2 * c->depth - 1 <= DS_GROUP && c->n_state >= 1, "decay_scan: bad rotation or depth");
  CA_REQUIRE(c->ldo >= c->H * c->vdim && c->ldp >= c->H * c->vdim && c->ldp >= c->H * c->dim, "decay_scan: rows too short");
  if (c->n_seq <= 0 || c->max_q_len <= 0) return CA_OK;
  CA_REQUIRE(c->n_seq <= 65535, "decay_scan: too many sequences");
  if (f32) return c->max_q_len == 1 ? decay_scan_launch<float, 1>(c, false, s) : decay_scan_launch<float, DS_GROUP>(c, false, s);
  if (c->max_q_len == 1) return decay_scan_launch<bf16, 1>(c, false, s);
  const bool chunked = chunkable(c, f32);
  CA_REQUIRE(!chunked || (c->chunks >= c->T / DC_TOK + c->n_seq + 1 && c->vp <= 256 && c->max_q_len <= 65535 * DC_TOK), "decay_scan: room for %d chunks is too little", c->chunks);
  const int rc = decay_scan_launch<bf16, DS_GROUP>(c, chunked, s);
  if (rc || !chunked) return rc;
  if (c->lower) return c->dim <= 64 ? chunk_launch<1, DECAY_FORGET>(c, s) : chunk_launch<2, DECAY_FORGET>(c, s);
  if (c->dim <= 64) return c->decay ? chunk_launch<1, DECAY_HEAD>(c, s) : chunk_launch<1, DECAY_LOW_RANK>(c, s);
  return c->decay ? chunk_launch<2, DECAY_HEAD>(c, s) : chunk_launch<2, DECAY_LOW_RANK>(c, s);
}

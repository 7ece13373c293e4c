// True fp32 linear layer (no reduced-precision matrix mode): Y[rows, N] = X[rows, K] W[g][N, K]^T, dense or grouped by the same device
// tile table as tc_gemm.cu.  For the all-fp32 mode of an engine (numerics checks), not for throughput: 64 x 64 output tiles, 256
// threads of 4 x 4 outputs, K in steps of 16 through shared memory, plain fused multiply-adds in K order.
// Reference counterpart: the fp32 linears of native/shared/cuda/linear.cu (cuBLAS there).
#define CA_PDL_CLASS 1
#include "common.cuh"

#define FL_T 64
#define FL_K 16

struct F32Args {
  const float* X; const float* W; float* Y;
  const int4* tiles; const int* n_tiles; const float* alpha;      // [G] output factors, or null
  int ldx, ldy, rows, N, K, act, grp_rows, grp_cols;      // act: 1 squared ReLU, 2 soft cap at act_p
  float act_p;
};

__global__ void __launch_bounds__(256) f32_linear_kernel(const F32Args a) {
  pdl_launch(); pdl_wait();
  __shared__ float xs[FL_K][FL_T + 4], ws[FL_K][FL_T + 4];
  int g = 0, row0 = 0, nrows = 0;
  if (a.tiles) {
    if ((int)blockIdx.y >= *a.n_tiles) return;
    const int4 t = a.tiles[blockIdx.y];
    g = t.x; row0 = t.y; nrows = min(t.z, a.rows - row0);
  } else {
    row0 = blockIdx.y * FL_T; nrows = min(FL_T, a.rows - row0);
  }
  const int n0 = blockIdx.x * FL_T, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const float* W = a.W + (size_t)g * a.N * a.K;
  // grouped tiles may hold more rows than a thread block covers: walk them
  for (int m0 = 0; m0 < nrows; m0 += FL_T) {
    float acc[4][4] = {};
    for (int k0 = 0; k0 < a.K; k0 += FL_K) {
      for (int i = tid; i < FL_T * FL_K; i += 256) {
        const int r = i / FL_K, k = i % FL_K;
        xs[k][r] = (m0 + r < nrows && k0 + k < a.K) ? a.X[(size_t)(row0 + m0 + r) * a.ldx + k0 + k] : 0.f;
        ws[k][r] = (n0 + r < a.N && k0 + k < a.K) ? W[(size_t)(n0 + r) * a.K + k0 + k] : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < FL_K; ++k) {
        float xv[4], wv[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) { xv[j] = xs[k][ty * 4 + j]; wv[j] = ws[k][tx * 4 + j]; }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = m0 + ty * 4 + i;
      if (r >= nrows) continue;
      const size_t o = a.grp_rows > 0 ? (size_t)(row0 + r - g * a.grp_rows) * a.ldy + (size_t)g * a.grp_cols : (size_t)(row0 + r) * a.ldy;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + tx * 4 + j;
        if (n >= a.N) continue;
        float v = a.alpha ? acc[i][j] * a.alpha[g] : acc[i][j];
        if (a.act == 1) { v = fmaxf(v, 0.f); v *= v; }
        if (a.act == 2) v = a.act_p * tanhf(v / a.act_p);
        a.Y[o + n] = v;
      }
    }
  }
}

extern "C" int cuteafd_f32_linear(const float* X, int ldx, const float* W, float* Y, int ldy, const void* tiles, const int* n_tiles, int max_tiles, int rows,
                                  int N, int K, int act, float act_p, int grp_rows, int grp_cols, const float* alpha, cudaStream_t s) {
  CA_REQUIRE(X && W && Y && (!tiles || (n_tiles && max_tiles > 0 && max_tiles <= 65535)) && act >= 0 && act <= 2 && (act != 2 || act_p > 0.f), "f32_linear: bad arguments");
  CA_REQUIRE(grp_rows == 0 || tiles, "f32_linear: token-major output belongs to a grouped product");
  if (rows <= 0 || N <= 0) return CA_OK;
  const F32Args a{X, W, Y, (const int4*)tiles, n_tiles, alpha, ldx, ldy, rows, N, K, act, grp_rows, grp_cols, act_p};
  const int m = tiles ? max_tiles : (rows + FL_T - 1) / FL_T;
  CA_REQUIRE(m <= 65535, "f32_linear: too many row tiles");
  CA_LAUNCH_PDL(f32_linear_kernel, dim3((N + FL_T - 1) / FL_T, m), 256, 0, s, a);
  CA_CHECK_LAUNCH("f32_linear");
  return CA_OK;
}

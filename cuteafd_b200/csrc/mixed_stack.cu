// Kernels of the mixed stacks: the token's part of a second table behind a layer.
//   side_gate        gelu_tanh(gate row) * the token's part of the table -> operand of the side projection
// T is the operand type: bf16, or float for the all-fp32 mode.  (No counterpart in the reference, which has no such family; norms and residual
// rows are hybrid_stack.cu's, attention, latents and HGRN2 the kernels of the other layer stacks.)
#include "stack_rows.cuh"

// table row of a token: `part` elements in all, this layer's from `col` on.
template <typename T>
__global__ void side_gate_kernel(const float* __restrict__ z, int ldz, const int* __restrict__ tokens, const bf16* __restrict__ table, int ldtab, int col, int n, int vocab, T* __restrict__ out,
                                 int ldo, int rows, int* status) {
  pdl_launch(); pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x, t = i / n, j = i % n;
  if (t >= rows) return;
  int tok = tokens[t];
  if (tok < 0 || tok >= vocab) { if (j == 0) ca_dev_fail(status, CA_DEV_BAD_INDEX, t); tok = 0; }
  const float v = z[(size_t)t * ldz + j], e = __bfloat162float(table[(size_t)tok * ldtab + col + j]);
  out[(size_t)t * ldo + j] = to_t<T>(0.5f * v * (1.f + tanhf(0.7978845608028654f * fmaf(0.044715f * v * v, v, v))) * e);
}

extern "C" int cuteafd_side_gate(const float* z, int ldz, const int* tokens, const void* table, int ldtab, int col, int n, int vocab, void* out, int ldo, int rows, int f32, int* status,
                                 cudaStream_t s) {
  CA_REQUIRE(z && tokens && table && out && n >= 1 && ldz >= n && ldo >= n && col >= 0 && col + n <= ldtab && vocab >= 1, "side_gate: bad arguments");
  if (rows <= 0) return CA_OK;
  const int grid = (int)(((long long)rows * n + 255) / 256);
  if (f32) CA_LAUNCH_PDL(side_gate_kernel<float>, grid, 256, 0, s, z, ldz, tokens, (const bf16*)table, ldtab, col, n, vocab, (float*)out, ldo, rows, status);
  else CA_LAUNCH_PDL(side_gate_kernel<bf16>, grid, 256, 0, s, z, ldz, tokens, (const bf16*)table, ldtab, col, n, vocab, (bf16*)out, ldo, rows, status);
  CA_CHECK_LAUNCH("side_gate");
  return CA_OK;
}

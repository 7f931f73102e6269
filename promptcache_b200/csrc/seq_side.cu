// The per-layer token-side input: a second embedding row of the token, gated by the stream and projected back into it.
//     u = W_gate x;   g = gelu(u) * e;   y = W_proj g;   x += y / sqrt(mean(y^2) + eps) * w          (e: this layer's part of the token's row)
//
// pcs_side_gate   g from u, between two library products (prompts).
#include "seq_common.cuh"

namespace pcs {

template <typename T>
__global__ void __launch_bounds__(256) side_gate_kernel(const T* __restrict__ u, long long u_stride, const T* __restrict__ table, long long table_stride,
                                                        int vocab, int col, const int64_t* __restrict__ ids, T* __restrict__ out, long long n, int dim) {
  const long long e = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (e >= n) return;
  const long long t = e / dim;
  const int c = static_cast<int>(e - t * dim);
  long long id = ids[t];
  if (id < 0 || id >= vocab) id = 0;
  const GluAct act(PCS_GLU_GELU_TANH);
  stf(out + e, act(ldf(u + t * u_stride + c), ldf(table + id * table_stride + col + c)));
}

}  // namespace pcs

PCS_API int pcs_side_gate(const void* u, int64_t u_stride, const void* table, int64_t table_stride, int vocab, int col, const int64_t* ids, void* out,
                          int n_tokens, int dim, int dtype, void* stream) {
  if (n_tokens == 0) return PCS_OK;
  PCS_REQUIRE(u && table && ids && out && n_tokens > 0 && dim > 0 && vocab > 0 && col >= 0 && col + dim <= table_stride && u_stride >= dim, "pcs_side_gate: bad arguments");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long n = static_cast<long long>(n_tokens) * dim;
  PCS_DISPATCH(dtype, pcs::side_gate_kernel<T><<<static_cast<unsigned>((n + 255) / 256), 256, 0, st>>>(static_cast<const T*>(u), u_stride, static_cast<const T*>(table),
                                                                                                          table_stride, vocab, col, ids, static_cast<T*>(out), n, dim));
  PCS_CHECK_CUDA(cudaGetLastError());
  pcs::count_launch();
  return PCS_OK;
}

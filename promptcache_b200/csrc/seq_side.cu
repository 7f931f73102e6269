// The per-layer token-side input: a second embedding row of the token, gated by the stream and projected back into it.
//     u = W_gate x;   g = gelu(u) * e;   y = W_proj g;   x += y / sqrt(mean(y^2) + eps) * w          (e: this layer's part of the token's row)
//
// pcs_side_gate       g from u, between two library products (prompts).
// pcs_side_boundary   a few tokens: the layer's residual sum in front of it and the next layer's norms behind it in the same launch.  A cluster of
//                     8 CTAs works on one token; a CTA owns an eighth of the columns of x, of W_gate and of the rows of W_proj (staged in
//                     shared memory while the first product runs).  What crosses between the CTAs goes through distributed
//                     shared memory: the partial sums of u, the sum of squares of y, the sum of squares of the new x.
#include <cooperative_groups.h>

#include "seq_common.cuh"
#include "seq_mma.cuh"

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

namespace cg = cooperative_groups;
constexpr int kSideCluster = 8, kSideThreads = 256, kSideRows = 8;   // rows of W_gate a warp has in flight

// VEC: width / 8, dim and every row are whole 16-byte pieces.  `stage`: this CTA's rows of W_proj fit the shared memory it was given.
template <typename T, bool VEC>
__global__ void __cluster_dims__(kSideCluster, 1, 1) __launch_bounds__(kSideThreads) side_boundary_kernel(const pcs_side_params p, int CW, int stage) {
  constexpr int N = Vec<T>::n;
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float red[33];
  __shared__ float sums[2];     // this CTA's sums of squares: y, new x
  cg::cluster_group cl = cg::this_cluster();
  const int rank = static_cast<int>(cl.block_rank()), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const long long t = blockIdx.y;
  const int W = p.width, dim = p.dim, c0 = rank * CW, cw = max(0, min(CW, W - c0));
  const int dimp = (dim + 3) & ~3;
  T* ps = reinterpret_cast<T*>(raw);                                        // [cw][dim + N]: rows one piece apart from whole banks
  float* xs = reinterpret_cast<float*>(raw + (stage ? static_cast<size_t>(CW) * (dim + N) * sizeof(T) : 0));   // [CW] the stream after the sublayers
  float* ys = xs + CW;          // [CW] W_proj g
  float* part = ys + CW;        // [dim] this CTA's share of u
  float* gs = part + dimp;      // [dim] the gated row
  const T* gate = static_cast<const T*>(p.gate) + c0;
  const T* proj = static_cast<const T*>(p.proj) + static_cast<long long>(c0) * dim;
  if (VEC && stage) {
    const int pieces = dim / N;
    for (int e = tid; e < cw * pieces; e += kSideThreads) {
      const int r = e / pieces, c = (e - r * pieces) * N;
      cp_async16(ps + r * (dim + N) + c, proj + static_cast<long long>(r) * dim + c);
    }
  }
  cp_async_commit();
  // u: a group of LPR lanes takes a row of this CTA's columns of W_gate, several rows in flight
  const int pieces = VEC ? cw / N : 1;
  int LPR = 32;
  if (VEC)
    while (LPR > 1 && LPR / 2 >= pieces) LPR /= 2;
  const int per = 32 / LPR, sub = lane / LPR, l0 = lane % LPR;   // rows side by side in a warp
  uint4 pre[kSideRows];
  if (VEC) {   // the first piece of the warp's first rows is requested before the stream's row
#pragma unroll
    for (int k = 0; k < kSideRows; ++k) {
      const int j = (warp + 8 * k) * per + sub;
      pre[k] = j < dim && l0 < pieces ? *reinterpret_cast<const uint4*>(gate + static_cast<long long>(j) * W + l0 * N) : make_uint4(0u, 0u, 0u, 0u);
    }
  }
  for (int c = tid; c < cw; c += kSideThreads) {
    float a = 0.f;
    for (int k = 0; k < p.n_y; ++k) a += ldf(static_cast<const T*>(p.y[k]) + t * p.y_stride[k] + c0 + c);
    xs[c] = p.x[t * W + c0 + c] + a;
  }
  __syncthreads();
  if (VEC) {
    auto fma_piece = [&](const uint4& w, int c, float& a) {
      float wv[N], xv[N];
      ld16(reinterpret_cast<const T*>(&w), wv);
      ldx(xs + c, xv);
#pragma unroll
      for (int e = 0; e < N; ++e) a = fmaf(wv[e], xv[e], a);
    };
    for (int j0 = warp; j0 * per < dim; j0 += 8 * kSideRows) {
      if (j0 != warp) {
#pragma unroll
        for (int k = 0; k < kSideRows; ++k) {
          const int j = (j0 + 8 * k) * per + sub;
          pre[k] = j < dim && l0 < pieces ? *reinterpret_cast<const uint4*>(gate + static_cast<long long>(j) * W + l0 * N) : make_uint4(0u, 0u, 0u, 0u);
        }
      }
#pragma unroll
      for (int k = 0; k < kSideRows; ++k) {
        const int j = (j0 + 8 * k) * per + sub;
        float a = 0.f;
        if (l0 < pieces) fma_piece(pre[k], l0 * N, a);
        if (j < dim)
          for (int q = l0 + LPR; q < pieces; q += LPR) fma_piece(*reinterpret_cast<const uint4*>(gate + static_cast<long long>(j) * W + q * N), q * N, a);
        for (int o = LPR / 2; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
        if (l0 == 0 && j < dim) part[j] = a;
      }
    }
  } else {
    for (int j = warp; j < dim; j += 8) {
      float a = 0.f;
      for (int c = lane; c < cw; c += 32) a = fmaf(ldf(gate + static_cast<long long>(j) * W + c), xs[c], a);
      a = warp_sum(a);
      if (lane == 0) part[j] = a;
    }
  }
  cp_async_wait<0>();
  cl.sync();
  {
    long long id = p.ids[t];
    if (id < 0 || id >= p.vocab) id = 0;
    const T* e = static_cast<const T*>(p.table) + id * p.table_stride + p.col;
    const GluAct act(PCS_GLU_GELU_TANH);
    for (int j = tid; j < dim; j += kSideThreads) {
      float u = 0.f;
#pragma unroll
      for (int r = 0; r < kSideCluster; ++r) u += cl.map_shared_rank(part, r)[j];
      gs[j] = act(u, ldf(e + j));
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < cw; c += kSideThreads) {
    float a0 = 0.f, a1 = 0.f;
    if (VEC) {
      const T* row = stage ? ps + c * (dim + N) : proj + static_cast<long long>(c) * dim;
#pragma unroll 4
      for (int j = 0; j < dim; j += N) {
        float wv[N], gv[N];
        ld16(row + j, wv);
        ldx(gs + j, gv);
#pragma unroll
        for (int e = 0; e < N; e += 2) {
          a0 = fmaf(wv[e], gv[e], a0);
          a1 = fmaf(wv[e + 1], gv[e + 1], a1);
        }
      }
    } else {
      for (int j = 0; j < dim; ++j) a0 = fmaf(ldf(proj + static_cast<long long>(c) * dim + j), gs[j], a0);
    }
    const float y = a0 + a1;
    ys[c] = y;
    ss = fmaf(y, y, ss);
  }
  ss = block_sum(ss, red);
  if (tid == 0) sums[0] = ss;
  cl.sync();
  float all = 0.f;
#pragma unroll
  for (int r = 0; r < kSideCluster; ++r) all += *cl.map_shared_rank(&sums[0], r);
  const float inv_y = 1.f / sqrtf(all / static_cast<float>(W) + p.eps);
  const T* nw = static_cast<const T*>(p.norm_w) + c0;
  const T* sv = p.step ? static_cast<const T*>(p.step) + c0 : nullptr;
  float sx = 0.f;
  for (int c = tid; c < cw; c += kSideThreads) {
    float a = ys[c] * inv_y * ldf(nw + c);
    if (p.x0) a += p.x0[t * W + c0 + c];
    if (sv) a += ldf(sv + c);
    const float v = xs[c] + a;
    xs[c] = v;
    p.x[t * W + c0 + c] = v;
    sx = fmaf(v, v, sx);
  }
  if (p.w1 || p.w2) {
    sx = block_sum(sx, red);
    if (tid == 0) sums[1] = sx;
    cl.sync();
    all = 0.f;
#pragma unroll
    for (int r = 0; r < kSideCluster; ++r) all += *cl.map_shared_rank(&sums[1], r);
    const float inv_x = 1.f / sqrtf(all / static_cast<float>(W) + p.eps);
    const T* w1 = static_cast<const T*>(p.w1);
    const T* w2 = static_cast<const T*>(p.w2);
    for (int c = tid; c < cw; c += kSideThreads) {
      const float v = xs[c] * inv_x;
      if (w1) stf(static_cast<T*>(p.h1) + t * W + c0 + c, v * (p.w_offset + ldf(w1 + c0 + c)));
      if (w2) stf(static_cast<T*>(p.h2) + t * W + c0 + c, v * (p.w_offset + ldf(w2 + c0 + c)));
    }
  }
  cl.sync();   // no CTA leaves while another may still read its sums
}

template <typename T, bool VEC>
static int launch_side_boundary(const pcs_side_params& p, int CW, int stage, size_t smem, cudaStream_t st) {
  PCS_CHECK_CUDA(cudaFuncSetAttribute(side_boundary_kernel<T, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
  side_boundary_kernel<T, VEC><<<dim3(kSideCluster, p.n_tokens), kSideThreads, smem, st>>>(p, CW, stage);
  PCS_CHECK_CUDA(cudaGetLastError());
  count_launch();
  return PCS_OK;
}

}  // namespace pcs

PCS_API int pcs_side_boundary(const pcs_side_params* p, void* stream) {
  PCS_REQUIRE(p, "pcs_side_boundary: null params");
  if (p->n_tokens == 0) return PCS_OK;
  PCS_REQUIRE(p->x && p->ids && p->table && p->gate && p->proj && p->norm_w, "pcs_side_boundary: null tensor");
  PCS_REQUIRE(p->n_y >= 0 && p->n_y <= 2 && (p->n_y < 1 || p->y[0]) && (p->n_y < 2 || p->y[1]), "pcs_side_boundary: at most two results, none of them null");
  PCS_REQUIRE((!p->w1 || p->h1) && (!p->w2 || p->h2), "pcs_side_boundary: a weight vector needs its output");
  PCS_REQUIRE(p->n_tokens > 0 && p->n_tokens <= 65535 && p->width > 0 && p->dim > 0 && p->vocab > 0 && p->col >= 0 && p->col + p->dim <= p->table_stride,
              "pcs_side_boundary: bad sizes");
  const int piece = p->dtype == PCS_BF16 ? 8 : 4, esz = p->dtype == PCS_BF16 ? 2 : 4;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = p->width % piece == 0 && p->dim % piece == 0 && al(p->gate) && al(p->proj);
  const int CW = ((p->width + pcs::kSideCluster - 1) / pcs::kSideCluster + 7) & ~7;
  const size_t base = (static_cast<size_t>(2) * CW + 2 * ((p->dim + 3) & ~3)) * sizeof(float);
  const size_t staged = base + static_cast<size_t>(CW) * (p->dim + piece) * esz;
  PCS_REQUIRE(base <= 200 * 1024, "pcs_side_boundary: width %d and dim %d exceed shared memory", p->width, p->dim);
  const int stage = vec && staged <= 200 * 1024 ? 1 : 0;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const size_t smem = stage ? staged : base;
  PCS_DISPATCH(p->dtype, {
    if (vec) return pcs::launch_side_boundary<T, true>(*p, CW, stage, smem, st);
    return pcs::launch_side_boundary<T, false>(*p, CW, stage, smem, st);
  });
  return PCS_OK;
}

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

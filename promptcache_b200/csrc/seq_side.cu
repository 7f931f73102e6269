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
constexpr int kSideCluster = 8, kSideThreads = 512, kSideWarps = kSideThreads / 32, kSideRows = 8;   // rows of W_gate a warp has in flight

// VEC: width and dim are whole 16-byte pieces and so is every row.  `stage`: this CTA's rows of W_proj fit the shared memory it was given.
// Everything that does not depend on another CTA is requested before the first sum: the rows of both matrices, this CTA's columns of the vectors,
// the token's row of the table.  What crosses between CTAs is PUSHED into every CTA's shared memory, so that after a cluster barrier each reads
// its own copy; sums are formed from the copies in the order of the CTAs.
template <typename T, bool VEC>
__global__ void __cluster_dims__(kSideCluster, 1, 1) __launch_bounds__(kSideThreads) side_boundary_kernel(const pcs_side_params p, int CW, int stage) {
  constexpr int N = Vec<T>::n;
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float sums[2][kSideCluster * kSideWarps];   // every warp's sum of squares, of every CTA: y, new x
  cg::cluster_group cl = cg::this_cluster();
  cl.barrier_arrive();          // (waited for before the first push: every CTA of the cluster runs by then)
  const int rank = static_cast<int>(cl.block_rank()), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const long long t = blockIdx.y;
  const int W = p.width, dim = p.dim, c0 = rank * CW, cw = max(0, min(CW, W - c0));
  const int dimp = (dim + 3) & ~3;
  T* ps = reinterpret_cast<T*>(raw);                                        // [cw][dim + N]: rows one piece apart from whole banks
  float* xs = reinterpret_cast<float*>(ps + (stage ? CW * (dim + N) : 0));  // [CW] the stream after the sublayers
  float* ys = xs + CW;          // [CW] W_proj g
  float* part = ys + CW;        // [cluster][dim] every CTA's share of u
  float* gs = part + kSideCluster * dimp;   // [dim] the token's row, then the gated row
  const T* gate = static_cast<const T*>(p.gate) + c0;
  const T* proj = static_cast<const T*>(p.proj) + static_cast<long long>(c0) * dim;
  long long id = p.ids[t];
  if (id < 0 || id >= p.vocab) id = 0;
  const T* nw = static_cast<const T*>(p.norm_w) + c0;
  const T* sv = p.step ? static_cast<const T*>(p.step) + c0 : nullptr;
  const T* w1 = p.w1 ? static_cast<const T*>(p.w1) + c0 : nullptr;
  const T* w2 = p.w2 ? static_cast<const T*>(p.w2) + c0 : nullptr;
  float* xg = p.x + t * W + c0;
  const float* x0 = p.x0 ? p.x0 + t * W + c0 : nullptr;
  const T* y0 = p.n_y > 0 ? static_cast<const T*>(p.y[0]) + t * p.y_stride[0] + c0 : nullptr;
  const T* y1 = p.n_y > 1 ? static_cast<const T*>(p.y[1]) + t * p.y_stride[1] + c0 : nullptr;
  // u: a group of LPR lanes takes a row of this CTA's columns of W_gate, several rows in flight
  const int pieces = VEC ? cw / N : 1;
  int LPR = 32;
  if (VEC)
    while (LPR > 1 && LPR / 2 >= pieces) LPR /= 2;
  const int per = 32 / LPR, sub = lane / LPR, l0 = lane % LPR;   // rows side by side in a warp
  uint4 pre[kSideRows];
  if (VEC) {
#pragma unroll
    for (int k = 0; k < kSideRows; ++k) {
      const int j = (warp + kSideWarps * k) * per + sub;
      pre[k] = j < dim && l0 < pieces ? *reinterpret_cast<const uint4*>(gate + static_cast<long long>(j) * W + l0 * N) : make_uint4(0u, 0u, 0u, 0u);
    }
  }
  // the thread's own column (rows wider than 8 * 512 read the others where they use them)
  float xv = 0.f, a0v = 0.f, a1v = 0.f, ent = 0.f, stv = 0.f, nv = 0.f, n1 = 0.f, n2 = 0.f;
  if (tid < cw) {
    xv = xg[tid];
    if (y0) a0v = ldf(y0 + tid);
    if (y1) a1v = ldf(y1 + tid);
    if (x0) ent = x0[tid];
    if (sv) stv = ldf(sv + tid);
    nv = ldf(nw + tid);
    if (w1) n1 = ldf(w1 + tid);
    if (w2) n2 = ldf(w2 + tid);
  }
  if (VEC) {
    if (stage) {
      const int pp = dim / N;
      for (int e = tid; e < cw * pp; e += kSideThreads) {
        const int r = e / pp, c = (e - r * pp) * N;
        cp_async16(ps + r * (dim + N) + c, proj + static_cast<long long>(r) * dim + c);
      }
    }
    cp_async_commit();
  }
  {
    const T* e = static_cast<const T*>(p.table) + id * p.table_stride + p.col;
    for (int j = tid; j < dim; j += kSideThreads) gs[j] = ldf(e + j);
  }
  if (tid < cw) xs[tid] = xv + (a0v + a1v);
  for (int c = tid + kSideThreads; c < cw; c += kSideThreads) xs[c] = xg[c] + ((y0 ? ldf(y0 + c) : 0.f) + (y1 ? ldf(y1 + c) : 0.f));
  __syncthreads();
  cl.barrier_wait();
  float* remote = cl.map_shared_rank(part, lane & (kSideCluster - 1)) + rank * dimp;   // where lane r pushes: CTA r's copy of this CTA's share
  if (VEC) {
    auto fma_piece = [&](const uint4& w, int c, float& a) {
      float wv[N], xv[N];
      ld16(reinterpret_cast<const T*>(&w), wv);
      ldx(xs + c, xv);
#pragma unroll
      for (int e = 0; e < N; ++e) a = fmaf(wv[e], xv[e], a);
    };
    for (int j0 = warp; j0 * per < dim; j0 += kSideWarps * kSideRows) {
      if (j0 != warp) {
#pragma unroll
        for (int k = 0; k < kSideRows; ++k) {
          const int j = (j0 + kSideWarps * k) * per + sub;
          pre[k] = j < dim && l0 < pieces ? *reinterpret_cast<const uint4*>(gate + static_cast<long long>(j) * W + l0 * N) : make_uint4(0u, 0u, 0u, 0u);
        }
      }
      float a[kSideRows];
#pragma unroll
      for (int k = 0; k < kSideRows; ++k) {
        const int j = (j0 + kSideWarps * k) * per + sub;
        a[k] = 0.f;
        if (l0 < pieces) fma_piece(pre[k], l0 * N, a[k]);
        if (j < dim)
          for (int q = l0 + LPR; q < pieces; q += LPR) fma_piece(*reinterpret_cast<const uint4*>(gate + static_cast<long long>(j) * W + q * N), q * N, a[k]);
      }
      for (int o = LPR / 2; o > 0; o >>= 1) {
#pragma unroll
        for (int k = 0; k < kSideRows; ++k) a[k] += __shfl_xor_sync(0xffffffffu, a[k], o);
      }
#pragma unroll
      for (int k = 0; k < kSideRows; ++k) {
        const int j = (j0 + kSideWarps * k) * per + sub;
        if (j < dim) {
          if (LPR >= kSideCluster) {   // (lane % 8 == l0 for the pushing lanes: their target is the mapped one)
            if (l0 < kSideCluster) remote[j] = a[k];
          } else {
            for (int r = l0; r < kSideCluster; r += LPR) cl.map_shared_rank(part, r)[rank * dimp + j] = a[k];
          }
        }
      }
    }
  } else {
    for (int j = warp; j < dim; j += kSideWarps) {
      float a = 0.f;
      for (int c = lane; c < cw; c += 32) a = fmaf(ldf(gate + static_cast<long long>(j) * W + c), xs[c], a);
      a = warp_sum(a);
      if (lane < kSideCluster) remote[j] = a;
    }
  }
  if (VEC) cp_async_wait<0>();
  cl.sync();
  {
    const GluAct act(PCS_GLU_GELU_TANH);
    for (int j = tid; j < dim; j += kSideThreads) {
      float u = 0.f;
#pragma unroll
      for (int r = 0; r < kSideCluster; ++r) u += part[r * dimp + j];
      gs[j] = act(u, gs[j]);
    }
  }
  __syncthreads();
  // every warp's sum of squares goes to all CTAs; after the barrier a warp adds all of them
  auto push = [&](int which, float v) {
    v = warp_sum(v);
    if (lane < kSideCluster) cl.map_shared_rank(&sums[which][0], lane)[rank * kSideWarps + warp] = v;
  };
  auto total = [&](int which) {
    float v = 0.f;
#pragma unroll
    for (int k = 0; k < kSideCluster * kSideWarps / 32; ++k) v += sums[which][lane + 32 * k];
    return warp_sum(v);
  };
  float ss = 0.f;
  if (VEC) {   // TPR neighbouring threads share a row of W_proj
    int TPR = 1;
    while (TPR < 8 && 2 * TPR * cw <= kSideThreads && 2 * TPR * N <= dim) TPR *= 2;
    const int h = tid & (TPR - 1);
    for (int cb = 0; cb < cw; cb += kSideThreads / TPR) {
      const int c = cb + tid / TPR;
      float a0 = 0.f, a1 = 0.f;
      if (c < cw) {
        const T* row = stage ? ps + c * (dim + N) : proj + static_cast<long long>(c) * dim;
#pragma unroll 4
        for (int j = h * N; j < dim; j += TPR * N) {
          float wv[N], gv[N];
          ld16(row + j, wv);
          ldx(gs + j, gv);
#pragma unroll
          for (int e = 0; e < N; e += 2) {
            a0 = fmaf(wv[e], gv[e], a0);
            a1 = fmaf(wv[e + 1], gv[e + 1], a1);
          }
        }
      }
      float y = a0 + a1;
      for (int o = 1; o < TPR; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (h == 0 && c < cw) {
        ys[c] = y;
        ss = fmaf(y, y, ss);
      }
    }
  } else {
    for (int c = tid; c < cw; c += kSideThreads) {
      float y = 0.f;
      for (int j = 0; j < dim; ++j) y = fmaf(ldf(proj + static_cast<long long>(c) * dim + j), gs[j], y);
      ys[c] = y;
      ss = fmaf(y, y, ss);
    }
  }
  push(0, ss);
  cl.sync();
  const float inv_y = 1.f / sqrtf(total(0) / static_cast<float>(W) + p.eps);
  float sx = 0.f;
  for (int c = tid; c < cw; c += kSideThreads) {
    const bool own = c == tid;
    float a = ys[c] * inv_y * (own ? nv : ldf(nw + c));
    if (x0) a += own ? ent : x0[c];
    if (sv) a += own ? stv : ldf(sv + c);
    const float v = xs[c] + a;
    xs[c] = v;
    xg[c] = v;
    sx = fmaf(v, v, sx);
  }
  if (p.w1 || p.w2) {
    push(1, sx);
    cl.sync();
    const float inv_x = 1.f / sqrtf(total(1) / static_cast<float>(W) + p.eps);
    for (int c = tid; c < cw; c += kSideThreads) {
      const float v = xs[c] * inv_x;
      const bool own = c == tid;
      if (w1) stf(static_cast<T*>(p.h1) + t * W + c0 + c, v * (p.w_offset + (own ? n1 : ldf(w1 + c))));
      if (w2) stf(static_cast<T*>(p.h2) + t * W + c0 + c, v * (p.w_offset + (own ? n2 : ldf(w2 + c))));
    }
  }
}   // (nothing is pushed after the last barrier, so a CTA may leave)

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
  const size_t base = (static_cast<size_t>(2) * CW + (pcs::kSideCluster + 1) * ((p->dim + 3) & ~3)) * sizeof(float);
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

// Residual sum with a norm in groups of channels, followed by a short causal convolution over time of the NEW stream (what the next
// sublayer reads where layers norm their results only) or by a grouped norm of it (the model's last norm).
//
// A token's convolution needs its taps - 1 predecessors' new stream rows.  Rows of the same step are being formed by other blocks,
// so a block forms the rows it needs again from the old stream and the sublayer's result (both are only read: the new stream
// goes to another buffer).  A block takes TB neighbouring tokens, so the rows it forms again are (taps - 1) / TB of its work; all
// rows' loads are requested before the one reduction that gives every (row, group) its root mean square.  Rows of earlier steps
// come from the slot's tail, kept twice (see seq_canon.cu).  Everything is 32-bit; h_out is rounded once, to the compute type.
#include "seq_common.cuh"

namespace pcs {

constexpr int kGnMaxTaps = 16;

// where a convolution's tail of a batch entry is read and written, and the token's place in its entry
struct TailView {
  int pos, pos0, len;
  const float* rd;   // rows: positions pos0 - R .. pos0 - 1
  float* wr;         // rows: positions pos0 + len - R .. pos0 + len - 1
};
__device__ __forceinline__ TailView tail_view(const pcs_gnconv_params& p, int t, int R) {
  TailView v;
  const int b = p.tok_seq[t];
  v.pos = p.tok_pos[t];
  v.pos0 = p.seq_pos0[b];
  v.len = p.seq_len[b];
  const int par = p.seq_par[b] & 1;
  float* base = p.tail + static_cast<long long>(p.seq_slot[b]) * 2 * R * p.width;
  v.rd = base + static_cast<long long>(par) * R * p.width;
  v.wr = base + static_cast<long long>(par ^ 1) * R * p.width;
  return v;
}

// Any sizes: one block per row; `inv` holds the factors 1 / rms of (row, predecessor) x group.
template <typename T>
__global__ void __launch_bounds__(256) gnconv_kernel(const pcs_gnconv_params p) {
  extern __shared__ float sm[];
  const int W = p.width, G = p.groups, S = W / G, R = p.conv_w ? p.taps - 1 : 0;
  const int r = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const long long row = p.rows ? p.rows[r] : r;
  float* inv = sm;                 // [R + 1][G]
  float* s0 = sm + (R + 1) * G;    // [width]: the row's new stream (next_w only)
  TailView tv{0, 0, 1, nullptr, nullptr};
  if (p.conv_w) tv = tail_view(p, r, R);
  const T* w = static_cast<const T*>(p.w);
  if (p.y) {
    for (int e = warp; e < (R + 1) * G; e += 8) {
      const int j = e / G, g = e - j * G;
      if (j > 0 && tv.pos - j < tv.pos0) continue;
      const T* y = static_cast<const T*>(p.y) + (row - j) * p.y_stride + g * S;
      float ss = 0.f;
      for (int i = lane; i < S; i += 32) { const float v = ldf(y + i); ss = fmaf(v, v, ss); }
      ss = warp_sum(ss);
      if (lane == 0) inv[e] = 1.f / sqrtf(ss / static_cast<float>(S) + p.eps);
    }
    __syncthreads();
  }
  auto fresh = [&](int j, int i) {  // channel i of the new stream of this step's row `row - j`
    float v = p.x[(row - j) * W + i];
    if (p.y) v = fmaf(ldf(static_cast<const T*>(p.y) + (row - j) * p.y_stride + i) * inv[j * G + i / S], ldf(w + i), v);
    return v;
  };
  T* h = static_cast<T*>(p.h_out) + static_cast<long long>(r) * W;
  const T* cw = static_cast<const T*>(p.conv_w);
  const int last_row = tv.pos - (tv.pos0 + tv.len - R);   // this token's row in the written tail, if >= 0
  for (int i = tid; i < W; i += 256) {
    const float v = fresh(0, i);
    if (p.x_out) p.x_out[row * W + i] = v;
    if (cw) {
      float acc = fmaf(v, ldf(cw + static_cast<long long>(R) * W + i), v);
      for (int j = 1; j <= R; ++j) {
        if (tv.pos - j < 0) break;
        const float vj = tv.pos - j >= tv.pos0 ? fresh(j, i) : tv.rd[static_cast<long long>(R - (tv.pos0 - (tv.pos - j))) * W + i];
        acc = fmaf(ldf(cw + static_cast<long long>(R - j) * W + i), vj, acc);
      }
      stf(h + i, acc);
      if (R > 0 && last_row >= 0) tv.wr[static_cast<long long>(last_row) * W + i] = v;
    } else if (p.next_w) {
      s0[i] = v;
    }
  }
  if (cw) {
    if (R > 0 && tv.pos == tv.pos0 + tv.len - 1 && tv.len < R)   // rows that stay: new row q is old row q + len
      for (int q = 0; q < R - tv.len; ++q)
        for (int i = tid; i < W; i += 256) tv.wr[static_cast<long long>(q) * W + i] = tv.rd[static_cast<long long>(q + tv.len) * W + i];
    return;
  }
  if (p.next_w == nullptr) return;
  __syncthreads();
  for (int g = warp; g < G; g += 8) {
    float ss = 0.f;
    for (int i = lane; i < S; i += 32) ss = fmaf(s0[g * S + i], s0[g * S + i], ss);
    ss = warp_sum(ss);
    if (lane == 0) inv[g] = 1.f / sqrtf(ss / static_cast<float>(S) + p.eps);
  }
  __syncthreads();
  const T* nw = static_cast<const T*>(p.next_w);
  for (int i = tid; i < W; i += 256) stf(h + i, s0[i] * inv[i / S] * ldf(nw + i));
}

// Sums over the runs of PG neighbouring pieces that form a norm group, for K rows at once: v[k] is this thread's piece of row k.  With
// one piece per thread and PG a power of two up to 32 the runs lie inside a warp and no shared memory is touched.
template <int K, int PPT>
__device__ __forceinline__ void group_sums(float (&v)[K][PPT], int NP, int PG, int G, float* ssq, float* tot) {
  const int tid = threadIdx.x, nthr = blockDim.x, warp = tid >> 5, lane = tid & 31;
  if (PPT == 1 && PG <= 32 && (PG & (PG - 1)) == 0) {
#pragma unroll
    for (int o = 1; o < 32; o <<= 1)
      if (o < PG) {
#pragma unroll
        for (int k = 0; k < K; ++k) v[k][0] += __shfl_xor_sync(0xffffffffu, v[k][0], o);
      }
    return;
  }
  __syncthreads();   // `ssq` may still be read from an earlier call
#pragma unroll
  for (int k = 0; k < K; ++k)
#pragma unroll
    for (int u = 0; u < PPT; ++u)
      if (tid + u * nthr < NP) ssq[k * NP + tid + u * nthr] = v[k][u];
  __syncthreads();
  for (int e = warp; e < K * G; e += nthr >> 5) {
    const int k = e / G, g = e - k * G;
    float a = 0.f;
    for (int i = lane; i < PG; i += 32) a += ssq[k * NP + g * PG + i];
    a = warp_sum(a);
    if (lane == 0) tot[e] = a;
  }
  __syncthreads();
#pragma unroll
  for (int u = 0; u < PPT; ++u) {
    const int pc = tid + u * nthr;
    if (pc < NP) {
#pragma unroll
      for (int k = 0; k < K; ++k) v[k][u] = tot[k * G + pc / PG];
    }
  }
}

// 16-byte pieces (the width, a group's width, strides and pointers are multiples of a piece; at most blockDim.x * PPT pieces per row).
// The block's rows are requested before it knows which of them its tokens need.
template <typename T, int PPT, int TB, int R>
__global__ void __launch_bounds__(256, (PPT == 1 ? 2 : 1)) gnconv_vec_kernel(const pcs_gnconv_params p) {
  constexpr int N = Vec<T>::n, RN = TB + R;   // rows a block may form: R predecessors, then its TB tokens
  extern __shared__ float sm[];
  const int W = p.width, G = p.groups, NP = W / N, PG = NP / G;
  const int t0 = blockIdx.x * TB, tid = threadIdx.x, nthr = blockDim.x;
  float* ssq = sm;            // [RN][NP]
  float* tot = sm + RN * NP;  // [RN][G]
  const T* cw = static_cast<const T*>(p.conv_w);
  // row k of the block is step row t0 - R + k (with `rows`: the listed row)
  float s[RN][PPT][N];
  uint4 yv[RN][PPT];
#pragma unroll
  for (int k = 0; k < RN; ++k) {
    const int r = t0 - R + k;
    const bool in = r >= 0 && r < p.n_rows;
    const long long row = in ? (p.rows ? p.rows[r] : r) : 0;
#pragma unroll
    for (int u = 0; u < PPT; ++u) {
      const int pc = tid + u * nthr;
      if (in && pc < NP) {
        ldx(p.x + row * W + pc * N, s[k][u]);
        if (p.y) yv[k][u] = *reinterpret_cast<const uint4*>(static_cast<const T*>(p.y) + row * p.y_stride + pc * N);
      } else {
#pragma unroll
        for (int e = 0; e < N; ++e) s[k][u][e] = 0.f;
        yv[k][u] = make_uint4(0u, 0u, 0u, 0u);
      }
    }
  }
  // few tokens: the weights are requested with the rows (many tokens: their loads are hidden by other blocks, the registers are not free)
  uint4 wq[PPT], cq[PPT][R + 1];
  if (TB == 1) {
#pragma unroll
    for (int u = 0; u < PPT; ++u) {
      const int pc = tid + u * nthr;
      if (pc < NP) {
        if (p.y) wq[u] = *reinterpret_cast<const uint4*>(static_cast<const T*>(p.w) + pc * N);
        if (cw) {
#pragma unroll
          for (int j = 0; j <= R; ++j) cq[u][j] = *reinterpret_cast<const uint4*>(cw + static_cast<long long>(R - j) * W + pc * N);
        }
      }
    }
  }
  // the tokens' places in their entries: how many of the R predecessors are rows of this step, and the tails
  int here[TB], before[TB], last_row[TB], shift[TB];   // predecessors in this step; predecessors at all; tail row to write; rows that stay move by this
  long long tail0[TB];                                 // element offset of the slot's copy that is read
  int par[TB];
  const T* w = static_cast<const T*>(p.w);
#pragma unroll
  for (int i = 0; i < TB; ++i) {
    here[i] = before[i] = 0;
    last_row[i] = -1;
    shift[i] = 0;
    tail0[i] = 0;
    par[i] = 0;
    if (R > 0 && cw && t0 + i < p.n_rows) {
      const int b = p.tok_seq[t0 + i], pos = p.tok_pos[t0 + i], pos0 = p.seq_pos0[b], len = p.seq_len[b];
      here[i] = min(R, pos - pos0);
      before[i] = min(R, pos);
      last_row[i] = pos - (pos0 + len - R);
      if (pos == pos0 + len - 1 && len < R) shift[i] = len;
      par[i] = p.seq_par[b] & 1;
      tail0[i] = (static_cast<long long>(p.seq_slot[b]) * 2 + par[i]) * R * W;
    }
  }
  auto unpack = [](const uint4& q, float (&o)[N]) { ld16(reinterpret_cast<const T*>(&q), o); };
  const float inv_n = 1.f / static_cast<float>(PG * N);
  if (p.y) {
    float ss[RN][PPT];
#pragma unroll
    for (int k = 0; k < RN; ++k)
#pragma unroll
      for (int u = 0; u < PPT; ++u) {
        float v[N], a = 0.f;
        unpack(yv[k][u], v);
#pragma unroll
        for (int e = 0; e < N; ++e) a = fmaf(v[e], v[e], a);
        ss[k][u] = a;
      }
    group_sums<RN, PPT>(ss, NP, PG, G, ssq, tot);
#pragma unroll
    for (int u = 0; u < PPT; ++u) {
      const int pc = tid + u * nthr;
      if (pc < NP) {
        float wv[N];
        if (TB == 1) unpack(wq[u], wv);
        else ld16(w + pc * N, wv);
#pragma unroll
        for (int k = 0; k < RN; ++k) {
          float v[N];
          unpack(yv[k][u], v);
          const float f = 1.f / sqrtf(fmaf(ss[k][u], inv_n, p.eps));
#pragma unroll
          for (int e = 0; e < N; ++e) s[k][u][e] = fmaf(v[e] * f, wv[e], s[k][u][e]);
        }
      }
    }
  }
#pragma unroll
  for (int u = 0; u < PPT; ++u) {
    const int pc = tid + u * nthr;
    if (pc < NP) {
#pragma unroll
      for (int i = 0; i < TB; ++i)
        if (t0 + i < p.n_rows) {
          if (p.x_out) stx(p.x_out + static_cast<long long>(p.rows ? p.rows[t0 + i] : t0 + i) * W + pc * N, s[R + i][u]);
          if (cw) {
            float o[N], wv[N];
            if (TB == 1) unpack(cq[u][0], wv);
            else ld16(cw + static_cast<long long>(R) * W + pc * N, wv);
#pragma unroll
            for (int e = 0; e < N; ++e) o[e] = fmaf(s[R + i][u][e], wv[e], s[R + i][u][e]);
#pragma unroll
            for (int j = 1; j <= R; ++j)
              if (j <= before[i]) {
                if (TB == 1) unpack(cq[u][j], wv);
                else ld16(cw + static_cast<long long>(R - j) * W + pc * N, wv);
                if (j <= here[i]) {
#pragma unroll
                  for (int e = 0; e < N; ++e) o[e] = fmaf(wv[e], s[R + i - j][u][e], o[e]);
                } else {   // position pos - j sits in tail row R - (pos0 - (pos - j)); pos - pos0 is `here` whenever it is below R
                  float q[N];
                  ldx(p.tail + tail0[i] + static_cast<long long>(R - (j - here[i])) * W + pc * N, q);
#pragma unroll
                  for (int e = 0; e < N; ++e) o[e] = fmaf(wv[e], q[e], o[e]);
                }
              }
            st16(static_cast<T*>(p.h_out) + static_cast<long long>(t0 + i) * W + pc * N, o);
            if (R > 0) {
              float* wr = p.tail + tail0[i] + (par[i] ? -1LL : 1LL) * R * W + pc * N;
              if (last_row[i] >= 0) stx(wr + static_cast<long long>(last_row[i]) * W, s[R + i][u]);
              if (shift[i] > 0)
                for (int q = 0; q < R - shift[i]; ++q) {
                  float v[N];
                  ldx(p.tail + tail0[i] + static_cast<long long>(q + shift[i]) * W + pc * N, v);
                  stx(wr + static_cast<long long>(q) * W, v);
                }
            }
          }
        }
    }
  }
  if (cw || p.next_w == nullptr) return;
  // the grouped norm of the new stream
  float ss[TB][PPT];
#pragma unroll
  for (int i = 0; i < TB; ++i)
#pragma unroll
    for (int u = 0; u < PPT; ++u) {
      float a = 0.f;
#pragma unroll
      for (int e = 0; e < N; ++e) a = fmaf(s[R + i][u][e], s[R + i][u][e], a);
      ss[i][u] = a;
    }
  group_sums<TB, PPT>(ss, NP, PG, G, ssq, tot);
#pragma unroll
  for (int u = 0; u < PPT; ++u) {
    const int pc = tid + u * nthr;
    if (pc < NP) {
      float nv[N];
      ld16(static_cast<const T*>(p.next_w) + pc * N, nv);
#pragma unroll
      for (int i = 0; i < TB; ++i)
        if (t0 + i < p.n_rows) {
          float o[N];
          const float f = 1.f / sqrtf(fmaf(ss[i][u], inv_n, p.eps));
#pragma unroll
          for (int e = 0; e < N; ++e) o[e] = s[R + i][u][e] * f * nv[e];
          st16(static_cast<T*>(p.h_out) + static_cast<long long>(t0 + i) * W + pc * N, o);
        }
    }
  }
}

template <typename T, int PPT, int TB, int R>
static int launch_gnconv_vec(const pcs_gnconv_params& p, cudaStream_t st) {
  const int np = p.width / Vec<T>::n, thr = PPT == 1 ? (np + 31) / 32 * 32 : 256;
  const size_t smem = static_cast<size_t>(TB + R) * (np + p.groups) * sizeof(float);
  gnconv_vec_kernel<T, PPT, TB, R><<<(p.n_rows + TB - 1) / TB, thr, smem, st>>>(p);
  PCS_CHECK_CUDA(cudaGetLastError());
  count_launch();
  return PCS_OK;
}

template <typename T, int R>
static int launch_gnconv_taps(const pcs_gnconv_params& p, cudaStream_t st) {
  const int np = p.width / Vec<T>::n;
  if (np > 256) return launch_gnconv_vec<T, 2, 1, R>(p, st);
  // four tokens per block where that leaves two blocks per SM
  if (R > 0 && p.n_rows >= 4 * 2 * 148) return launch_gnconv_vec<T, 1, (R > 0 ? 4 : 1), R>(p, st);
  return launch_gnconv_vec<T, 1, 1, R>(p, st);
}

template <typename T>
static int launch_gnconv(const pcs_gnconv_params& p, cudaStream_t st, bool vec) {
  const int R = p.conv_w ? p.taps - 1 : 0;
  if (vec) {
    if (R == 0) return launch_gnconv_taps<T, 0>(p, st);
    if (R == 1) return launch_gnconv_taps<T, 1>(p, st);
    if (R == 2) return launch_gnconv_taps<T, 2>(p, st);
    if (R == 3) return launch_gnconv_taps<T, 3>(p, st);
  }
  const size_t smem = (static_cast<size_t>(R + 1) * p.groups + p.width) * sizeof(float);
  PCS_REQUIRE(smem <= 200 * 1024, "pcs_group_norm_conv: width %d with %d groups exceeds shared memory", p.width, p.groups);
  if (smem > 48 * 1024) PCS_CHECK_CUDA(cudaFuncSetAttribute(gnconv_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
  gnconv_kernel<T><<<p.n_rows, 256, smem, st>>>(p);
  PCS_CHECK_CUDA(cudaGetLastError());
  count_launch();
  return PCS_OK;
}

}  // namespace pcs

PCS_API int pcs_group_norm_conv(const pcs_gnconv_params* p, void* stream) {
  PCS_REQUIRE(p, "pcs_group_norm_conv: null params");
  if (p->n_rows == 0) return PCS_OK;
  PCS_REQUIRE(p->x && p->n_rows > 0 && p->width > 0 && p->groups > 0 && p->width % p->groups == 0, "pcs_group_norm_conv: %d groups do not divide width %d", p->groups,
              p->width);
  PCS_REQUIRE(p->y == nullptr || p->w, "pcs_group_norm_conv: the result's norm needs its weight");
  PCS_REQUIRE(!(p->conv_w && p->next_w), "pcs_group_norm_conv: either the convolution or the next norm");
  PCS_REQUIRE((p->conv_w == nullptr && p->next_w == nullptr) || p->h_out, "pcs_group_norm_conv: null h_out");
  if (p->conv_w) {
    PCS_REQUIRE(p->rows == nullptr && p->taps >= 1 && p->taps <= pcs::kGnMaxTaps, "pcs_group_norm_conv: taps %d outside 1..%d, or a row subset", p->taps, pcs::kGnMaxTaps);
    PCS_REQUIRE((p->tail || p->taps == 1) && p->tok_seq && p->tok_pos && p->seq_slot && p->seq_pos0 && p->seq_len && p->seq_par,
                "pcs_group_norm_conv: the convolution needs the tail and the batch description");
    PCS_REQUIRE(p->y == nullptr || p->x_out != p->x, "pcs_group_norm_conv: the new stream must not overwrite the old one under a convolution");
  }
  const int piece = p->dtype == PCS_BF16 ? 8 : 4;
  const long long esz = p->dtype == PCS_BF16 ? 2 : 4;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = p->impl != 1 && p->width % piece == 0 && (p->width / p->groups) % piece == 0 && p->width <= 512 * piece && p->groups <= 64 && al(p->x) && al(p->x_out) &&
                   al(p->y) && (p->y_stride * esz) % 16 == 0 && al(p->w) && al(p->next_w) && al(p->conv_w) && al(p->tail) && al(p->h_out);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  PCS_DISPATCH(p->dtype, return pcs::launch_gnconv<T>(*p, st, vec));
}

// Gated delta rule over the slot pool.
//
// Per head, with a decay per key channel (or one per head, formed here from its pre-activation) and a step size beta in (0, 1):
//     S <- diag(decay_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t          (S: dim x vdim, 32-bit)
// q, k and v come out of a short causal convolution with silu; q and k are unit vectors per head.
//
// pcs_short_conv        the convolution over time per channel, silu, unit vectors.  Inputs of earlier steps sit in the slot's tail,
//                       kept twice so that the copy a step reads is never the one it writes.
// pcs_delta_inputs      decoding: the convolution and the two low-rank products beside it (decays, output gate) in one launch.
// pcs_delta_scan        token by token.  The columns of S evolve independently given k, q and the decays, so the grid covers
//                       (sequence, head, slice of columns): state in registers (dim <= 256, aligned) or in shared memory.
// pcs_delta_chunk_prep  prompts: everything about a chunk of 64 tokens that does not need the state it starts from.
// pcs_delta_chunk_scan  prompts: the chunks in order, two products per chunk on a slice of columns held in shared memory.
// pcs_delta_chunk_out   prompts in bfloat16: the read-out of the chunks with the per-head norm and gate.
// pcs_head_norm_gate    per-head norm and sigmoid (or silu) gate of the recurrence's result.
#include "seq_common.cuh"
#include "seq_mma.cuh"

namespace pcs {

// ---- short convolution ---------------------------------------------------------------------------------------------------------
constexpr int kScMaxTaps = 16;

struct ConvPlace {
  int pos, pos0, len;
  const float* rd;   // tail rows: positions pos0 - R .. pos0 - 1
  float* wr;         // tail rows: positions pos0 + len - R .. pos0 + len - 1
};
__device__ __forceinline__ ConvPlace conv_place(const pcs_shortconv_params& p, int t, int R, int C) {
  ConvPlace v;
  const int b = p.tok_seq[t];
  v.pos = p.tok_pos[t];
  v.pos0 = p.seq_pos0[b];
  v.len = p.seq_len[b];
  const int par = p.seq_par[b] & 1;
  float* base = p.tail + static_cast<long long>(p.seq_slot[b]) * 2 * R * C;
  v.rd = base + static_cast<long long>(par) * R * C;
  v.wr = base + static_cast<long long>(par ^ 1) * R * C;
  return v;
}

__device__ __forceinline__ float silu_(float z) { return z * sigmoidf_(z); }

// log of a head's decay from its pre-activation
__device__ __forceinline__ float head_log_decay(float z, float rate) { return -rate * softplusf_(z); }

// Any sizes: one block per token; a warp per query / key head, then the value channels.
template <typename T>
__global__ void __launch_bounds__(256) short_conv_kernel(const pcs_shortconv_params p) {
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = p.dim, U = 2 * p.kv_heads * D, C = U + p.v_width, R = p.taps - 1;
  const ConvPlace cp = conv_place(p, t, R, C);
  const T* x = static_cast<const T*>(p.proj) + static_cast<long long>(t) * p.row_stride + p.c_off;
  const T* cw = static_cast<const T*>(p.conv_w);
  const int last_row = cp.pos - (cp.pos0 + cp.len - R);
  auto value = [&](int c) {
    float acc = ldf(cw + static_cast<long long>(R) * C + c) * ldf(x + c);
    for (int j = 1; j <= R; ++j) {
      if (cp.pos - j < 0) break;
      const float v = cp.pos - j >= cp.pos0 ? ldf(x - static_cast<long long>(j) * p.row_stride + c)
                                            : cp.rd[static_cast<long long>(R - (cp.pos0 - (cp.pos - j))) * C + c];
      acc = fmaf(ldf(cw + static_cast<long long>(R - j) * C + c), v, acc);
    }
    return silu_(acc);
  };
  float* qk = p.qk_out + static_cast<long long>(t) * U;
  for (int hd = warp; hd < 2 * p.kv_heads; hd += 8) {
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) { const float v = value(hd * D + d); ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    const float f = (hd < p.kv_heads ? p.q_scale : 1.f) / sqrtf(ss + p.unit_eps);
    for (int d = lane; d < D; d += 32) qk[hd * D + d] = value(hd * D + d) * f;
  }
  T* vo = static_cast<T*>(p.v_out) + static_cast<long long>(t) * p.v_width;
  for (int c = tid; c < p.v_width; c += 256) stf(vo + c, value(U + c));
  if (R > 0 && last_row >= 0)
    for (int c = tid; c < C; c += 256) cp.wr[static_cast<long long>(last_row) * C + c] = ldf(x + c);
  if (R > 0 && cp.pos == cp.pos0 + cp.len - 1 && cp.len < R)
    for (int q = 0; q < R - cp.len; ++q)
      for (int c = tid; c < C; c += 256) cp.wr[static_cast<long long>(q) * C + c] = cp.rd[static_cast<long long>(q + cp.len) * C + c];
}

// 16-byte pieces: a thread owns one piece of the channels [blockIdx.y * CB, ...) for TB neighbouring tokens, whose rows and R predecessors are
// requested before the block knows which of them its tokens need.  CB is a multiple of dim, so a head's pieces meet in this block: by
// shuffles where a head is a power of two up to 32 pieces, else through shared memory.
template <typename T, int TB, int R>
__device__ __forceinline__ void short_conv_tile(const pcs_shortconv_params& p, int CB) {
  constexpr int N = Vec<T>::n, RN = TB + R;
  __shared__ float ssq[TB][256];
  const int t0 = blockIdx.x * TB, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = p.dim, U = 2 * p.kv_heads * D, C = U + p.v_width;
  const int c_lo = blockIdx.y * CB, c = c_lo + tid * N;
  const bool active = tid * N < CB && c < C;
  const T* cw = static_cast<const T*>(p.conv_w);
  uint4 xv[RN];
  const T* x = static_cast<const T*>(p.proj) + p.c_off + c;
#pragma unroll
  for (int k = 0; k < RN; ++k) {
    const int r = t0 - R + k;
    xv[k] = active && r >= 0 && r < p.n_tokens ? *reinterpret_cast<const uint4*>(x + static_cast<long long>(r) * p.row_stride) : make_uint4(0u, 0u, 0u, 0u);
  }
  uint4 cq[R + 1];   // (many tokens: other blocks hide these loads)
  if (TB == 1 && active) {
#pragma unroll
    for (int j = 0; j <= R; ++j) cq[j] = *reinterpret_cast<const uint4*>(cw + static_cast<long long>(R - j) * C + c);
  }
  // the tokens' places in their entries (see the boundary kernel): predecessors in this step and at all, tail row to write, rows that stay
  int here[TB], before[TB], last_row[TB], shift[TB], par[TB];
  long long tail0[TB];
#pragma unroll
  for (int i = 0; i < TB; ++i) {
    here[i] = before[i] = shift[i] = par[i] = 0;
    last_row[i] = -1;
    tail0[i] = 0;
    if (R > 0 && t0 + i < p.n_tokens) {
      const int b = p.tok_seq[t0 + i], pos = p.tok_pos[t0 + i], pos0 = p.seq_pos0[b], len = p.seq_len[b];
      here[i] = min(R, pos - pos0);
      before[i] = min(R, pos);
      last_row[i] = pos - (pos0 + len - R);
      if (pos == pos0 + len - 1 && len < R) shift[i] = len;
      par[i] = p.seq_par[b] & 1;
      tail0[i] = (static_cast<long long>(p.seq_slot[b]) * 2 + par[i]) * R * C + c;
    }
  }
  float o[TB][N], ss[TB];
#pragma unroll
  for (int i = 0; i < TB; ++i) {
    ss[i] = 0.f;
#pragma unroll
    for (int e = 0; e < N; ++e) o[i][e] = 0.f;
  }
  if (active) {
#pragma unroll
    for (int j = 0; j <= R; ++j) {
      float wv[N];
      if (TB == 1) ld16(reinterpret_cast<const T*>(&cq[j]), wv);
      else ld16(cw + static_cast<long long>(R - j) * C + c, wv);
#pragma unroll
      for (int i = 0; i < TB; ++i)
        if (j <= before[i]) {
          float v[N];
          if (j <= here[i]) ld16(reinterpret_cast<const T*>(&xv[R + i - j]), v);
          else ldx(p.tail + tail0[i] + static_cast<long long>(R - (j - here[i])) * C, v);
#pragma unroll
          for (int e = 0; e < N; ++e) o[i][e] = fmaf(wv[e], v[e], o[i][e]);
        }
    }
#pragma unroll
    for (int i = 0; i < TB; ++i) {
#pragma unroll
      for (int e = 0; e < N; ++e) {
        o[i][e] = silu_(o[i][e]);
        ss[i] = fmaf(o[i][e], o[i][e], ss[i]);
      }
      if (R > 0) {
        float* wr = p.tail + tail0[i] + (par[i] ? -1LL : 1LL) * R * C;
        float v[N];
        if (last_row[i] >= 0) {
          ld16(reinterpret_cast<const T*>(&xv[R + i]), v);
          stx(wr + static_cast<long long>(last_row[i]) * C, v);
        }
        if (shift[i] > 0)
          for (int q = 0; q < R - shift[i]; ++q) {
            ldx(p.tail + tail0[i] + static_cast<long long>(q + shift[i]) * C, v);
            stx(wr + static_cast<long long>(q) * C, v);
          }
      }
    }
  }
  // every piece's head sum
  const int PD = D / N;
  if (c_lo < U) {   // (uniform) this block holds query or key heads
    if (PD <= 32 && (PD & (PD - 1)) == 0) {
#pragma unroll
      for (int q = 1; q < 32; q <<= 1)
        if (q < PD) {
#pragma unroll
          for (int i = 0; i < TB; ++i) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], q);
        }
    } else {
#pragma unroll
      for (int i = 0; i < TB; ++i) ssq[i][tid] = ss[i];
      __syncthreads();
      const int heads = min(CB, U - c_lo) / D;
      // a warp adds the pieces of one (token, head); the sum goes to the head's first piece
      for (int e = warp; e < TB * heads; e += static_cast<int>(blockDim.x) >> 5) {
        const int i = e / heads, hd = e - i * heads;
        float a = 0.f;
        for (int k = lane; k < PD; k += 32) a += ssq[i][hd * PD + k];
        a = warp_sum(a);
        if (lane == 0) ssq[i][hd * PD] = a;
      }
      __syncthreads();
      if (c < U) {
#pragma unroll
        for (int i = 0; i < TB; ++i) ss[i] = ssq[i][tid / PD * PD];
      }
    }
  }
  if (!active) return;
#pragma unroll
  for (int i = 0; i < TB; ++i)
    if (t0 + i < p.n_tokens) {
      if (c < U) {
        const float f = (c < U / 2 ? p.q_scale : 1.f) / sqrtf(ss[i] + p.unit_eps);
#pragma unroll
        for (int e = 0; e < N; ++e) o[i][e] *= f;
        stx(p.qk_out + static_cast<long long>(t0 + i) * U + c, o[i]);
      } else {
        st16(static_cast<T*>(p.v_out) + static_cast<long long>(t0 + i) * p.v_width + (c - U), o[i]);
      }
    }
}

template <typename T, int TB, int R>
__global__ void __launch_bounds__(256, 2) short_conv_vec_kernel(const pcs_shortconv_params p, int CB) {
  short_conv_tile<T, TB, R>(p, CB);
}

// Few tokens (decoding): the convolution, and behind its blocks in blockIdx.y the two low-rank products that read the same projection
// row, the decays and the output gate's pre-activation: 8 lanes per output, 16-byte pieces of the matrix row where it is aligned.
template <typename T, int R>
__global__ void __launch_bounds__(256) delta_inputs_kernel(const pcs_shortconv_params p, const pcs_lowrank_params q, int CB, int ny) {
  if (static_cast<int>(blockIdx.y) < ny) {
    short_conv_tile<T, 1, R>(p, CB);
    return;
  }
  constexpr int N = Vec<T>::n;
  const int t = blockIdx.x, lane8 = threadIdx.x & 7, HD = q.heads * q.dim, n_out = HD + q.gate_width;
  const int o = (static_cast<int>(blockIdx.y) - ny) * (blockDim.x >> 3) + (threadIdx.x >> 3);
  const bool ok = o < n_out, dec = o < HD;
  const int rank = dec ? q.decay_rank : q.gate_rank, row = dec ? o : o - HD;
  const T* w = static_cast<const T*>(dec ? q.a2 : q.g2) + static_cast<long long>(row) * rank;
  const T* x = static_cast<const T*>(p.proj) + static_cast<long long>(t) * p.row_stride + (dec ? q.a_off : q.g_off);
  float acc = 0.f;
  if (ok) {
    const bool vec = rank % N == 0 && ((reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(x)) & 15) == 0;
    if (vec) {
      for (int r = lane8 * N; r < rank; r += 8 * N) {
        float a[N], b[N];
        ld16(w + r, a);
        ld16(x + r, b);
#pragma unroll
        for (int e = 0; e < N; ++e) acc = fmaf(a[e], b[e], acc);
      }
    } else {
      for (int r = lane8; r < rank; r += 8) acc = fmaf(ldf(w + r), ldf(x + r), acc);
    }
  }
#pragma unroll
  for (int m = 1; m < 8; m <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, m);
  if (!ok || lane8 != 0) return;
  if (dec) q.decay_out[static_cast<long long>(t) * HD + o] = expf(-q.rate[o / q.dim] * softplusf_(acc + q.dt_bias[o]));
  else stf(static_cast<T*>(q.gate_out) + static_cast<long long>(t) * q.gate_width + row, acc);
}

template <typename T, int R>
static void launch_short_conv_taps(const pcs_shortconv_params& p, const pcs_lowrank_params* q, cudaStream_t st) {
  const int per = 256 * Vec<T>::n, C = 2 * p.kv_heads * p.dim + p.v_width;
  int CB = per / p.dim * p.dim;
  if (p.n_tokens < 64 || q) {   // few tokens: narrow channel blocks, so that the launch covers more SMs
    const int small = (32 * Vec<T>::n + p.dim - 1) / p.dim * p.dim;
    if (small < CB) CB = small;
  }
  const int ny = (C + CB - 1) / CB;
  int thr = (CB / Vec<T>::n + 31) / 32 * 32;
  if (q) {
    if (thr < 128) thr = 128;
    const int outs = q->heads * q->dim + q->gate_width, extra = (outs + thr / 8 - 1) / (thr / 8);
    delta_inputs_kernel<T, R><<<dim3(p.n_tokens, ny + extra), thr, 0, st>>>(p, *q, CB, ny);
  } else if (R > 0 && p.n_tokens >= 4 * 148) {
    short_conv_vec_kernel<T, (R > 0 ? 4 : 1), R><<<dim3((p.n_tokens + 3) / 4, ny), thr, 0, st>>>(p, CB);
  } else {
    short_conv_vec_kernel<T, 1, R><<<dim3(p.n_tokens, ny), thr, 0, st>>>(p, CB);
  }
}

template <typename T>
static int launch_short_conv(const pcs_shortconv_params& p, const pcs_lowrank_params* q, cudaStream_t st, bool vec) {
  if (!vec) short_conv_kernel<T><<<p.n_tokens, 256, 0, st>>>(p);
  else if (p.taps == 1) launch_short_conv_taps<T, 0>(p, q, st);
  else if (p.taps == 2) launch_short_conv_taps<T, 1>(p, q, st);
  else if (p.taps == 3) launch_short_conv_taps<T, 2>(p, q, st);
  else launch_short_conv_taps<T, 3>(p, q, st);
  PCS_CHECK_CUDA(cudaGetLastError());
  count_launch();
  return PCS_OK;
}

// ---- token by token --------------------------------------------------------------------------------------------------------------
// Any sizes: S of VS columns in shared memory, thread (r, c) owns rows r, r + R, ... of column c.
template <typename T>
__global__ void __launch_bounds__(1024) delta_scan_kernel(const pcs_delta_params p, int VS, int R) {
  extern __shared__ float sm[];
  const int D = p.dim, V = p.vdim, H = p.heads, U = 2 * p.kv_heads * D;
  const int v0 = blockIdx.z * VS, vs = min(VS, V - v0);
  float* S = sm;               // [D][VS]
  float* ks = S + D * VS;      // [D]
  float* qs = ks + D;          // [D]
  float* as = qs + D;          // [D]
  float* us = as + D;          // [VS]
  float* part = us + VS;       // [R][VS]
  const int b = blockIdx.x, head = blockIdx.y, hk = head / (H / p.kv_heads), tid = threadIdx.x, nthr = blockDim.x;
  const int slot = p.seq_slot[b], len = p.seq_len[b], off = p.seq_off[b];
  if (len <= 0) return;
  const bool fresh = p.seq_pos0[b] == 0;
  float* Sg = p.s_pool + (static_cast<long long>(slot) * H + head) * D * V;
  for (int e = tid; e < D * vs; e += nthr) {
    const int d = e / vs, c = e - d * vs;
    S[d * VS + c] = fresh ? 0.f : Sg[static_cast<long long>(d) * V + v0 + c];
  }
  const int c = tid % VS, r = tid / VS;
  const bool active = r < R && c < vs;
  __syncthreads();
  for (int i = 0; i < len; ++i) {
    const long long t = off + i;
    for (int d = tid; d < D; d += nthr) {
      qs[d] = p.qk[t * U + hk * D + d];
      ks[d] = p.qk[t * U + (p.kv_heads + hk) * D + d];
      as[d] = p.decay ? p.decay[t * (static_cast<long long>(H) * D) + head * D + d]
                      : expf(head_log_decay(ldf(static_cast<const T*>(p.a) + t * p.a_stride + head) + p.dt_bias[head], p.rate[head]));
    }
    __syncthreads();
    if (active) {
      float num = 0.f;
      for (int d = r; d < D; d += R) {
        const float sv = as[d] * S[d * VS + c];
        S[d * VS + c] = sv;
        num = fmaf(sv, ks[d], num);
      }
      part[r * VS + c] = num;
    }
    __syncthreads();
    if (tid < vs) {
      float a = 0.f;
      for (int rr = 0; rr < R; ++rr) a += part[rr * VS + tid];
      const float beta = sigmoidf_(ldf(static_cast<const T*>(p.b) + t * p.b_stride + head));
      us[tid] = beta * (ldf(static_cast<const T*>(p.v) + t * (static_cast<long long>(H) * V) + head * V + v0 + tid) - a);
    }
    __syncthreads();
    if (active) {
      const float u = us[c];
      float num = 0.f;
      for (int d = r; d < D; d += R) {
        const float sv = fmaf(ks[d], u, S[d * VS + c]);
        S[d * VS + c] = sv;
        num = fmaf(sv, qs[d], num);
      }
      part[r * VS + c] = num;
    }
    __syncthreads();
    if (tid < vs) {
      float o = 0.f;
      for (int rr = 0; rr < R; ++rr) o += part[rr * VS + tid];
      p.o[t * (static_cast<long long>(H) * V) + head * V + v0 + tid] = o;
    }
    __syncthreads();
  }
  for (int e = tid; e < D * vs; e += nthr) {
    const int d = e / vs, cc = e - d * vs;
    Sg[static_cast<long long>(d) * V + v0 + cc] = S[d * VS + cc];
  }
}

constexpr int kDsRing = 12;   // shared-memory slots of tokens whose q / k / decays are in flight or waiting
constexpr int kDsAhead = 8;   // tokens requested ahead of the arithmetic
constexpr int kDsGroup = 4;   // tokens computed between two block barriers

// State in registers.  A warp owns 8 columns; lane = 8 * rg + c: column c, rows 4 (rg + 4 m) + e for m < M, e < 4 (four row groups
// share a column, so a column's sums are two shuffles).  One pass over the decayed state gives both S^T k and S^T q; the read-out
// after the write is then S^T q + (k . q) u.  Rows past dim hold zeros.  The order of every sum is fixed by M alone.  HD: one decay per
// head, formed here from its pre-activation (requested a group ahead, like the step sizes).
template <typename T, int M, bool HD>
__global__ void __launch_bounds__(256) delta_scan_reg_kernel(const pcs_delta_params p, int W) {
  extern __shared__ __align__(16) float ring[];   // per slot: q[16 M] k[16 M] decay[16 M] (per channel)
  constexpr int DP = 16 * M, NR = HD ? 2 : 3;
  const int D = p.dim, V = p.vdim, H = p.heads, U = 2 * p.kv_heads * D;
  const int b = blockIdx.x, head = blockIdx.y, hk = head / (H / p.kv_heads), v0 = blockIdx.z * 8 * W;
  const int tid = threadIdx.x, nthr = blockDim.x, warp = tid >> 5, lane = tid & 31, rg = lane >> 3;
  const int slot = p.seq_slot[b], len = p.seq_len[b], off = p.seq_off[b];
  if (len <= 0) return;
  const bool fresh = p.seq_pos0[b] == 0;
  const int col = v0 + warp * 8 + (lane & 7);
  const bool okc = col < V;
  const int cd = D / 4;
  auto issue = [&](int i) {
    const long long t = off + i;
    float* s = ring + (i % kDsRing) * NR * DP;
    for (int e = tid; e < NR * (DP / 4); e += nthr) {
      const int which = e / (DP / 4), c = e - which * (DP / 4);
      float* dst = s + which * DP + c * 4;
      if (c < cd) {
        const float* src = which == 0 ? p.qk + t * U + hk * D : which == 1 ? p.qk + t * U + (p.kv_heads + hk) * D : p.decay + t * (static_cast<long long>(H) * D) + head * D;
        cp_async16(dst, src + c * 4);
      } else {
        *reinterpret_cast<float4*>(dst) = make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
  };
  for (int i = 0; i < kDsAhead; ++i) {
    if (i < len) issue(i);
    cp_async_commit();
  }
  float* Sg = p.s_pool + (static_cast<long long>(slot) * H + head) * D * V;
  float S[M][4];
#pragma unroll
  for (int m = 0; m < M; ++m)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = 4 * (rg + 4 * m) + e;
      S[m][e] = (!fresh && d < D && okc) ? Sg[static_cast<long long>(d) * V + col] : 0.f;
    }
  const T* vg = static_cast<const T*>(p.v) + static_cast<long long>(off) * H * V + head * V + col;
  const T* bg = static_cast<const T*>(p.b) + static_cast<long long>(off) * p.b_stride + head;
  const T* ag = HD ? static_cast<const T*>(p.a) + static_cast<long long>(off) * p.a_stride + head : nullptr;
  const float a_bias = HD ? p.dt_bias[head] : 0.f, a_rate = HD ? p.rate[head] : 0.f;
  float vn[kDsGroup], bn[kDsGroup], an[kDsGroup];   // the next group's values and step sizes, requested a group ahead
#pragma unroll
  for (int u = 0; u < kDsGroup; ++u) {
    vn[u] = (u < len && okc) ? ldf(vg + static_cast<long long>(u) * H * V) : 0.f;
    bn[u] = u < len ? ldf(bg + u * p.b_stride) : 0.f;
    an[u] = HD && u < len ? ldf(ag + u * p.a_stride) : 0.f;
  }
  for (int i0 = 0; i0 < len; i0 += kDsGroup) {
    cp_async_wait<kDsAhead - kDsGroup>();
    __syncthreads();
    float vc[kDsGroup], bc[kDsGroup], ac[kDsGroup];
#pragma unroll
    for (int u = 0; u < kDsGroup; ++u) {
      vc[u] = vn[u];
      bc[u] = bn[u];
      ac[u] = an[u];
      const int nx = i0 + kDsGroup + u;
      vn[u] = (nx < len && okc) ? ldf(vg + static_cast<long long>(nx) * H * V) : 0.f;
      bn[u] = nx < len ? ldf(bg + nx * p.b_stride) : 0.f;
      an[u] = HD && nx < len ? ldf(ag + nx * p.a_stride) : 0.f;
      if (i0 + kDsAhead + u < len) issue(i0 + kDsAhead + u);
      cp_async_commit();
    }
#pragma unroll
    for (int u = 0; u < kDsGroup; ++u) {
      const int i = i0 + u;
      if (i >= len) break;
      const float* cur = ring + (i % kDsRing) * NR * DP;
      const float hd = HD ? expf(head_log_decay(ac[u] + a_bias, a_rate)) : 0.f;
      float pk = 0.f, pq = 0.f, kq = 0.f;
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int d = 4 * (rg + 4 * m);
        const float4 q = *reinterpret_cast<const float4*>(cur + d), k = *reinterpret_cast<const float4*>(cur + DP + d),
                     a = HD ? make_float4(hd, hd, hd, hd) : *reinterpret_cast<const float4*>(cur + 2 * DP + d);
        S[m][0] *= a.x; S[m][1] *= a.y; S[m][2] *= a.z; S[m][3] *= a.w;
        pk = fmaf(S[m][0], k.x, fmaf(S[m][1], k.y, fmaf(S[m][2], k.z, fmaf(S[m][3], k.w, pk))));
        pq = fmaf(S[m][0], q.x, fmaf(S[m][1], q.y, fmaf(S[m][2], q.z, fmaf(S[m][3], q.w, pq))));
        kq = fmaf(k.x, q.x, fmaf(k.y, q.y, fmaf(k.z, q.z, fmaf(k.w, q.w, kq))));
      }
#pragma unroll
      for (int o = 8; o <= 16; o <<= 1) {
        pk += __shfl_xor_sync(0xffffffffu, pk, o);
        pq += __shfl_xor_sync(0xffffffffu, pq, o);
        kq += __shfl_xor_sync(0xffffffffu, kq, o);
      }
      const float un = sigmoidf_(bc[u]) * (vc[u] - pk);
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const float4 k = *reinterpret_cast<const float4*>(cur + DP + 4 * (rg + 4 * m));
        S[m][0] = fmaf(k.x, un, S[m][0]); S[m][1] = fmaf(k.y, un, S[m][1]); S[m][2] = fmaf(k.z, un, S[m][2]); S[m][3] = fmaf(k.w, un, S[m][3]);
      }
      if (rg == 0 && okc) p.o[(static_cast<long long>(off) + i) * H * V + head * V + col] = fmaf(kq, un, pq);
    }
  }
#pragma unroll
  for (int m = 0; m < M; ++m)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int d = 4 * (rg + 4 * m) + e;
      if (d < D && okc) Sg[static_cast<long long>(d) * V + col] = S[m][e];
    }
}

// ---- in chunks -------------------------------------------------------------------------------------------------------------------
// A chunk's 64 rows form four blocks of 16.  With B the running sums of the log decays, r(I) the row before block I:
//   pairs inside a block take the exact factor exp(B_i - B_s) channel by channel;
//   pairs across blocks (row i of block I, row s of block J < I) factor it into exp(B_i - B_r(I)) * exp(B_r(I) - B_r(J+1)) * exp(B_r(J+1) - B_s):
//   every exponent is <= 0, and each factor is at least their product, so nothing is lost that the product does not lose.
// So q and k are scaled in place to their block's start and the keys to their block's end, and the pairs across blocks are plain products.
constexpr int kC = PCS_DELTA_CHUNK, kCB = 16, kNB = kC / kCB;
constexpr int kDpThreads = 384;

__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// hi keeps the sign, the exponent and 10 bits of the fraction; the remainder is exact in 32-bit and its own leading bits are what the unit reads
__device__ __forceinline__ void split_tf32(float x, uint32_t& hi, uint32_t& lo) {
  hi = __float_as_uint(x) & 0xffffe000u;
  lo = __float_as_uint(x - __uint_as_float(hi));
}

__device__ __forceinline__ int delta_kd_slot(int d) { return (d & ~63) + 4 * (d & 15) + ((d & 63) >> 4); }

// M x = rhs by forward substitution, one column per thread, the column in registers: first the dim columns of diag(beta) K exp(B), then the
// vdim columns of diag(beta) V.  `key(i, col)` gives row i of column col of K exp(B).
template <typename T, typename Key>
__device__ __forceinline__ void delta_chunk_solve(const pcs_delta_chunk_params& p, const float* As, const float* beta, long long base, int first, int n, int head, Key key) {
  const int D = p.dim, V = p.vdim, H = p.heads, tid = threadIdx.x;
  float* wg = p.w + base * ((D + 7) & ~7) * kC;
  float* ug = p.u + base * kC * V;
#pragma unroll 1
  for (int col = tid; col < D + V; col += kDpThreads) {
    float x[kC];
    long long v_step = static_cast<long long>(H) * V, u_step = V;
    asm volatile("" : "+l"(v_step), "+l"(u_step));   // (64 row offsets each, taken out of the column loop, would spill)
    if (col < D) {
#pragma unroll
      for (int i = 0; i < kC; ++i) x[i] = beta[i] * key(i, col);
    } else {
      const T* v = static_cast<const T*>(p.v) + static_cast<long long>(first) * H * V + head * V + (col - D);
#pragma unroll
      for (int i = 0; i < kC; ++i) x[i] = i < n ? beta[i] * ldf(v + i * v_step) : 0.f;
    }
#pragma unroll
    for (int i = 1; i < kC; ++i) {
      float a0 = 0.f, a1 = 0.f;
#pragma unroll
      for (int j = 0; j < i; j += 4) {
        const float4 a = *reinterpret_cast<const float4*>(As + i * kC + j);   // (entries from i on are zero)
        a0 = fmaf(a.x, x[j], a0);
        if (j + 1 < i) a1 = fmaf(a.y, x[j + 1], a1);
        if (j + 2 < i) a0 = fmaf(a.z, x[j + 2], a0);
        if (j + 3 < i) a1 = fmaf(a.w, x[j + 3], a1);
      }
      x[i] -= a0 + a1;
    }
    if (col < D) {
      float* o = wg + static_cast<long long>(col) * kC;
#pragma unroll
      for (int r = 0; r < 16; ++r) *reinterpret_cast<float4*>(o + 4 * r) = make_float4(x[r], x[r + 16], x[r + 32], x[r + 48]);
    } else {
#pragma unroll
      for (int i = 0; i < kC; ++i) ug[i * u_step + (col - D)] = x[i];
    }
  }
}

// The same in bfloat16 runs: M^-1 is formed once (a unit lower triangular 64 x 64 matrix: its four diagonal blocks of 16 by substitution, one
// column per thread, then the blocks below them, diagonal by diagonal, all in 32-bit multiply-adds), and both results are products
// M^-1 X with TF32 hi + lo operands, w written as the scan's operand fragments.  `inv` [64][kTi] shared memory.
constexpr int kTi = kC + 4;

template <typename Key>
__device__ __forceinline__ void delta_chunk_solve_tc(const pcs_delta_chunk_params& p, const float* As, const float* beta, float* inv, long long base, int first, int n,
                                                     int head, Key key) {
  const int D = p.dim, V = p.vdim, H = p.heads, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  for (int e = tid; e < kC * kC; e += kDpThreads) {
    const int i = e >> 6, j = e & 63;
    if ((i >> 4) != (j >> 4)) inv[i * kTi + j] = 0.f;
  }
  if (tid < kC) {
    const int b0 = tid & ~15, c = tid & 15;
    float x[kCB];
#pragma unroll
    for (int i = 0; i < kCB; ++i) {
      float a = 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) a = fmaf(As[(b0 + i) * kC + b0 + j], x[j], a);
      x[i] = (i == c ? 1.f : 0.f) - a;    // (zero above the diagonal by itself)
    }
#pragma unroll
    for (int i = 0; i < kCB; ++i) inv[(b0 + i) * kTi + b0 + c] = x[i];
  }
  __syncthreads();
#pragma unroll 1
  for (int d = 1; d < kNB; ++d) {   // blocks (I, I - d): first sum_K A[I, K] inv[K, J], kept in place, then -inv[I, I] times it
    const int cnt = (kNB - d) * kCB * kCB;
    for (int e = tid; e < cnt; e += kDpThreads) {
      const int I = (e >> 8) + d, J = I - d, i = I * kCB + ((e >> 4) & 15), j = J * kCB + (e & 15);
      float a0 = 0.f, a1 = 0.f;
      for (int q = J * kCB; q < I * kCB; q += 2) {
        a0 = fmaf(As[i * kC + q], inv[q * kTi + j], a0);
        a1 = fmaf(As[i * kC + q + 1], inv[(q + 1) * kTi + j], a1);
      }
      inv[i * kTi + j] = a0 + a1;
    }
    __syncthreads();
    float r[(kNB - 1) * kCB * kCB / kDpThreads];   // (two outputs per thread on the first diagonal)
#pragma unroll
    for (int m = 0; m < (kNB - 1) * kCB * kCB / kDpThreads; ++m) {
      const int e = tid + m * kDpThreads;
      r[m] = 0.f;
      if (e < cnt) {
        const int I = (e >> 8) + d, i = (e >> 4) & 15, j = (I - d) * kCB + (e & 15);
        float a0 = 0.f, a1 = 0.f;
#pragma unroll
        for (int q = 0; q < kCB; q += 2) {
          a0 = fmaf(inv[(I * kCB + i) * kTi + I * kCB + q], inv[(I * kCB + q) * kTi + j], a0);
          a1 = fmaf(inv[(I * kCB + i) * kTi + I * kCB + q + 1], inv[(I * kCB + q + 1) * kTi + j], a1);
        }
        r[m] = -(a0 + a1);
      }
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < (kNB - 1) * kCB * kCB / kDpThreads; ++m) {
      const int e = tid + m * kDpThreads;
      if (e < cnt) {
        const int I = (e >> 8) + d;
        inv[(I * kCB + ((e >> 4) & 15)) * kTi + (I - d) * kCB + (e & 15)] = r[m];
      }
    }
    __syncthreads();
  }
  // A warp and round takes 32 columns as four tiles of 8, of w or of u.  Which column a tile's place stands for is free: in a tile of w place x is
  // channel (x >> 1) + 4 (x & 1), so that a lane's accumulators are its operand fragment of the scan's w S; of u's 32 columns place x of tile q is
  // column 4 x + q, so that a lane's four values of a row, read or written, are neighbours.
  const int D8 = (D + 7) & ~7, NW = D8 / 8, GW = (NW + 3) / 4, groups = GW + (V + 31) / 32;
  float* wg = p.w + base * D8 * kC;
  float* ug = p.u + base * kC * V;
  const __nv_bfloat16* vb = static_cast<const __nv_bfloat16*>(p.v) + static_cast<long long>(first) * H * V + head * V;
  const bool quads = (V & 3) == 0 && (reinterpret_cast<uintptr_t>(p.v) & 7) == 0;
#pragma unroll 1
  for (int grp = warp; grp < groups; grp += kDpThreads / 32) {
    const bool of_w = grp < GW;
    const int t0 = grp * 4, cu = (grp - GW) * 32 + 4 * g;   // first tile of w; this lane's four columns of u
    uint2 vr[kC / 8][2];
    if (!of_w) {   // the lane's values of all steps, requested at once
#pragma unroll
      for (int ks = 0; ks < kC / 8; ++ks)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int i = 8 * ks + t + 4 * h;
          const __nv_bfloat16* r = vb + static_cast<long long>(i) * H * V + cu;
          vr[ks][h] = make_uint2(0u, 0u);
          if (i < n) {
            if (quads) {
              if (cu < V) vr[ks][h] = *reinterpret_cast<const uint2*>(r);
            } else {
              float x[4];
#pragma unroll
              for (int q = 0; q < 4; ++q) x[q] = cu + q < V ? ldf(r + q) : 0.f;
              vr[ks][h] = make_uint2(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]));
            }
          }
        }
    }
    float acc[4][4][4];
#pragma unroll
    for (int a = 0; a < 4; ++a)
#pragma unroll
      for (int b = 0; b < 4; ++b) acc[a][b][0] = acc[a][b][1] = acc[a][b][2] = acc[a][b][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < kC / 8; ++ks) {
      uint32_t bh[4][2], bl[4][2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int i = 8 * ks + t + 4 * h;
        const float bt = beta[i];
        float x[4];
        if (of_w) {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int c = 8 * (t0 + q) + (g >> 1) + 4 * (g & 1);
            x[q] = c < D ? key(i, c) : 0.f;
          }
        } else {
          x[0] = __uint_as_float(vr[ks][h].x << 16);
          x[1] = __uint_as_float(vr[ks][h].x & 0xffff0000u);
          x[2] = __uint_as_float(vr[ks][h].y << 16);
          x[3] = __uint_as_float(vr[ks][h].y & 0xffff0000u);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) split_tf32(bt * x[q], bh[q][h], bl[q][h]);
      }
#pragma unroll
      for (int mt = ks / 2; mt < 4; ++mt) {   // (row tiles above the diagonal hold zeros)
        const float* a = inv + (16 * mt + g) * kTi + 8 * ks + t;
        uint32_t ah[4], al[4];
        split_tf32(a[0], ah[0], al[0]);
        split_tf32(a[8 * kTi], ah[1], al[1]);
        split_tf32(a[4], ah[2], al[2]);
        split_tf32(a[8 * kTi + 4], ah[3], al[3]);
#pragma unroll
        for (int q = 0; q < 4; ++q) mma_tf32(acc[q][mt], ah, bh[q][0], bh[q][1]);
#pragma unroll
        for (int q = 0; q < 4; ++q) mma_tf32(acc[q][mt], ah, bl[q][0], bl[q][1]);
#pragma unroll
        for (int q = 0; q < 4; ++q) mma_tf32(acc[q][mt], al, bh[q][0], bh[q][1]);
      }
    }
    if (of_w) {
#pragma unroll
      for (int q = 0; q < 4; ++q)
        if (t0 + q < NW) {
#pragma unroll
          for (int mt = 0; mt < 4; ++mt)
            *reinterpret_cast<float4*>(wg + ((static_cast<long long>(t0 + q) * 4 + mt) * 32 + lane) * 4) = make_float4(acc[q][mt][0], acc[q][mt][2], acc[q][mt][1], acc[q][mt][3]);
        }
    } else {
#pragma unroll
      for (int mt = 0; mt < 4; ++mt)
#pragma unroll
        for (int x = 0; x < 4; ++x) {   // place 2 t + (x & 1) of row 16 mt + g + 8 (x >> 1)
          const int c = (grp - GW) * 32 + 4 * (2 * t + (x & 1));
          float* o = ug + static_cast<long long>(16 * mt + g + 8 * (x >> 1)) * V + c;
          if (quads) {
            if (c < V) *reinterpret_cast<float4*>(o) = make_float4(acc[0][mt][x], acc[1][mt][x], acc[2][mt][x], acc[3][mt][x]);
          } else {
#pragma unroll
            for (int q = 0; q < 4; ++q)
              if (c + q < V) o[q] = acc[q][mt][x];
          }
        }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(kDpThreads) delta_chunk_prep_kernel(const pcs_delta_chunk_params p) {
  extern __shared__ __align__(16) float sm[];
  const int D = p.dim, V = p.vdim, H = p.heads, D4 = (D + 3) & ~3, DP = D4 + 4, U = 2 * p.kv_heads * D, L = (D + 63) & ~63;
  float* qs = sm;              // [64][DP]: q, later scaled to its block's start
  float* ks = qs + kC * DP;    // [64][DP]: k, later scaled to its block's start
  float* Bs = ks + kC * DP;    // [64][DP]: running sums, later the keys scaled to their block's end; at last [64][kTi]
  float* f1 = Bs + kC * (DP > kTi ? DP : kTi);    // [D4] each: the running sums at the blocks' ends, later exp(B_r(1)), exp(B_r(2) - B_r(1)), exp(B_r(3) - B_r(2))
  float* f2 = f1 + D4;
  float* f3 = f2 + D4;
  float* fe = f3 + D4;
  float* As = fe + D4;         // [64][64] beta_i A[i, s]
  float* beta = As + kC * kC;  // [64]
  const int cn = blockIdx.x, head = blockIdx.y, hk = head / (H / p.kv_heads), tid = threadIdx.x;
  const int first = p.chunk_first[cn], n = p.chunk_len[cn];
  const long long base = static_cast<long long>(cn) * H + head;
  // bfloat16 runs work in the base-2 domain (exponential unit, relative error near 2^-22), float32 runs with the library exponential
  constexpr bool kFast = sizeof(T) == 2;
  constexpr float kLog = kFast ? 1.4426950408889634f : 1.f;
  auto ex = [](float x) { return kFast ? ex2(x) : expf(x); };
  const int warp = tid >> 5, lane = tid & 31;
  constexpr int kWarps = kDpThreads / 32;
  {
    const float* qb = p.qk + hk * D;
    const float* kb = p.qk + (p.kv_heads + hk) * D;
    const float* lb = p.ld + head * D;
    const bool vec = D == D4 && ((reinterpret_cast<uintptr_t>(p.qk) | reinterpret_cast<uintptr_t>(p.ld)) & 15) == 0;
    if (vec) {   // a warp takes a row at a time, the rows' loads overlap
      for (int d = lane * 4; d < D; d += 128) {
#pragma unroll
        for (int it = 0; it < (kC + kWarps - 1) / kWarps; ++it) {
          const int i = warp + it * kWarps;
          if (i >= kC) break;
          float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q, l = q;
          if (i < n) {
            const long long t = first + i;
            q = *reinterpret_cast<const float4*>(qb + t * U + d);
            k = *reinterpret_cast<const float4*>(kb + t * U + d);
            l = *reinterpret_cast<const float4*>(lb + t * (static_cast<long long>(H) * D) + d);
          }
          *reinterpret_cast<float4*>(qs + i * DP + d) = q;
          *reinterpret_cast<float4*>(ks + i * DP + d) = k;
          *reinterpret_cast<float4*>(Bs + i * DP + d) = make_float4(l.x * kLog, l.y * kLog, l.z * kLog, l.w * kLog);
        }
      }
    } else {
      for (int i = warp; i < kC; i += kWarps)
        for (int d = lane; d < D4; d += 32) {
          const long long t = first + i;
          const bool ok = i < n && d < D;
          qs[i * DP + d] = ok ? qb[t * U + d] : 0.f;
          ks[i * DP + d] = ok ? kb[t * U + d] : 0.f;
          Bs[i * DP + d] = ok ? lb[t * (static_cast<long long>(H) * D) + d] * kLog : 0.f;
        }
    }
  }
  if (tid < kC) beta[tid] = tid < n ? sigmoidf_(ldf(static_cast<const T*>(p.b) + static_cast<long long>(first + tid) * p.b_stride + head)) : 0.f;
  for (int e = tid; e < kC * kC; e += kDpThreads) As[e] = 0.f;
  float* ag = p.a + base * kC * kC;
  for (int e = tid; e < kC * kC; e += kDpThreads)
    if ((e & 63) > (e >> 6)) ag[e] = 0.f;   // above the diagonal
  __syncthreads();
  for (int d = tid; d < D4; d += kDpThreads) {
    float acc = 0.f;
#pragma unroll 8
    for (int i = 0; i < kC; ++i) {
      acc += Bs[i * DP + d];
      Bs[i * DP + d] = acc;
    }
  }
  __syncthreads();
  // pairs inside the blocks: (block, i, s <= i), 136 per block, every pair by four neighbouring threads that split the channels
  for (int e = tid >> 2; e < kNB * 136; e += kDpThreads / 4) {
    const int blk = e / 136, pr = e - blk * 136;
    int i = static_cast<int>((sqrtf(8.f * pr + 1.f) - 1.f) * 0.5f);
    while ((i + 1) * (i + 2) / 2 <= pr) ++i;
    while (i * (i + 1) / 2 > pr) --i;
    const int s = blk * kCB + (pr - i * (i + 1) / 2);
    i += blk * kCB;
    float aq = 0.f, ak = 0.f;
    for (int d = (tid & 3) * 4; d < D4; d += 16) {
      const float4 bi = *reinterpret_cast<const float4*>(Bs + i * DP + d), bs = *reinterpret_cast<const float4*>(Bs + s * DP + d);
      const float4 qi = *reinterpret_cast<const float4*>(qs + i * DP + d), ki = *reinterpret_cast<const float4*>(ks + i * DP + d);
      const float4 k4 = *reinterpret_cast<const float4*>(ks + s * DP + d);
      const float x0 = k4.x * ex(bi.x - bs.x), x1 = k4.y * ex(bi.y - bs.y), x2 = k4.z * ex(bi.z - bs.z), x3 = k4.w * ex(bi.w - bs.w);
      aq = fmaf(qi.x, x0, fmaf(qi.y, x1, fmaf(qi.z, x2, fmaf(qi.w, x3, aq))));
      ak = fmaf(ki.x, x0, fmaf(ki.y, x1, fmaf(ki.z, x2, fmaf(ki.w, x3, ak))));
    }
    const unsigned grp = 0xfu << (tid & 28);
    aq += __shfl_xor_sync(grp, aq, 1);
    ak += __shfl_xor_sync(grp, ak, 1);
    aq += __shfl_xor_sync(grp, aq, 2);
    ak += __shfl_xor_sync(grp, ak, 2);
    if ((tid & 3) == 0) {
      ag[i * kC + s] = aq;
      if (s < i) As[i * kC + s] = beta[i] * ak;
    }
  }
  __syncthreads();
  // the running sums at the blocks' ends, then per (token, channel): what leaves the chunk, q and k scaled to their block's start, and in
  // place of the running sums the keys scaled to their block's end (the last block's keys meet no later block)
  for (int d = tid; d < D4; d += kDpThreads) {
    f1[d] = Bs[15 * DP + d];
    f2[d] = Bs[31 * DP + d];
    f3[d] = Bs[47 * DP + d];
    fe[d] = Bs[63 * DP + d];
  }
  __syncthreads();
  {
    float* qd = p.qd + base * kC * D;
    float* kd = p.kd + base * kC * L;
    if (kFast) {   // the outgoing keys as fragments: a warp takes (16 channels, 8 tokens) at a time and writes 512 bytes
      for (int f = warp; f < (L / 16) * (kC / 8); f += kWarps) {
        const int mt = f >> 3, kt = f & 7;
        float o[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          const int i = kt * 8 + (lane & 3) + 4 * (r >> 1), d = mt * 16 + (lane >> 2) + 8 * (r & 1);
          o[r] = d < D ? ks[i * DP + d] * ex(fe[d] - Bs[i * DP + d]) : 0.f;
        }
        *reinterpret_cast<float4*>(kd + (static_cast<long long>(f) * 32 + lane) * 4) = make_float4(o[0], o[1], o[2], o[3]);
      }
      __syncthreads();
    }
    for (int i = warp; i < kC; i += kWarps) {
#pragma unroll 4
      for (int d = lane; d < D4; d += 32) {
        const int o = i * DP + d;
        const float bv = Bs[o], q = qs[o], k = ks[o];
        const float br = i < 16 ? 0.f : i < 32 ? f1[d] : i < 48 ? f2[d] : f3[d];
        const float bn = i < 16 ? f1[d] : i < 32 ? f2[d] : i < 48 ? f3[d] : bv;
        const float es = ex(bv - br);
        if (d < D) {
          qd[i * D + d] = q * ex(bv);
          if (!kFast) kd[static_cast<long long>(i) * L + delta_kd_slot(d)] = k * ex(fe[d] - bv);
        }
        qs[o] = q * es;
        ks[o] = k * es;
        Bs[o] = k * ex(bn - bv);
      }
    }
    for (int e = kFast ? kC * L : tid; e < kC * (L - D); e += kDpThreads) {   // the padding of the outgoing keys
      const int i = e / (L - D), d = D + (e - i * (L - D));
      kd[static_cast<long long>(i) * L + delta_kd_slot(d)] = 0.f;
    }
  }
  __syncthreads();
  for (int d = tid; d < D4; d += kDpThreads) {
    const float b1 = f1[d], b2 = f2[d], b3 = f3[d];
    f1[d] = ex(b1);
    f2[d] = ex(b2 - b1);
    f3[d] = ex(b3 - b2);
    if (d < D) p.g[base * D + d] = ex(fe[d]);
  }
  __syncthreads();
  // pairs across blocks: six (I, J) pairs of 16 x 16, 2 x 2 pairs per thread
  for (int e = tid; e < 6 * 64; e += kDpThreads) {
    const int pr = e >> 6, q4 = e & 63;
    const int I = pr == 0 ? 1 : pr < 3 ? 2 : 3, J = pr == 0 ? 0 : pr < 3 ? pr - 1 : pr - 3;
    const int i = I * kCB + (q4 >> 3), s = J * kCB + (q4 & 7);   // rows i, i + 8 and keys s, s + 8
    const float* g1 = J + 1 < I ? (J == 0 ? f2 : f3) : nullptr;   // from the end of J to the start of I: one block between
    const float* g2 = J + 2 < I ? f3 : nullptr;                    // or two
    float q00 = 0.f, q01 = 0.f, q10 = 0.f, q11 = 0.f, k00 = 0.f, k01 = 0.f, k10 = 0.f, k11 = 0.f;
    for (int d = 0; d < D4; d += 4) {
      float4 ka = *reinterpret_cast<const float4*>(Bs + s * DP + d), kb = *reinterpret_cast<const float4*>(Bs + (s + 8) * DP + d);
      if (g1) {
        const float4 f = *reinterpret_cast<const float4*>(g1 + d);
        ka.x *= f.x; ka.y *= f.y; ka.z *= f.z; ka.w *= f.w;
        kb.x *= f.x; kb.y *= f.y; kb.z *= f.z; kb.w *= f.w;
      }
      if (g2) {
        const float4 f = *reinterpret_cast<const float4*>(g2 + d);
        ka.x *= f.x; ka.y *= f.y; ka.z *= f.z; ka.w *= f.w;
        kb.x *= f.x; kb.y *= f.y; kb.z *= f.z; kb.w *= f.w;
      }
      auto dot = [](const float4& a, const float4& b, float c) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, c)))); };
      const float4 qa = *reinterpret_cast<const float4*>(qs + i * DP + d), qb = *reinterpret_cast<const float4*>(qs + (i + 8) * DP + d);
      q00 = dot(qa, ka, q00); q01 = dot(qa, kb, q01); q10 = dot(qb, ka, q10); q11 = dot(qb, kb, q11);
      const float4 xa = *reinterpret_cast<const float4*>(ks + i * DP + d), xb = *reinterpret_cast<const float4*>(ks + (i + 8) * DP + d);
      k00 = dot(xa, ka, k00); k01 = dot(xa, kb, k01); k10 = dot(xb, ka, k10); k11 = dot(xb, kb, k11);
    }
    ag[i * kC + s] = q00; ag[i * kC + s + 8] = q01; ag[(i + 8) * kC + s] = q10; ag[(i + 8) * kC + s + 8] = q11;
    As[i * kC + s] = beta[i] * k00; As[i * kC + s + 8] = beta[i] * k01;
    As[(i + 8) * kC + s] = beta[i + 8] * k10; As[(i + 8) * kC + s + 8] = beta[i + 8] * k11;
  }
  __syncthreads();
  auto key = [&](int i, int col) {
    const float e1 = f1[col];
    return ks[i * DP + col] * (i < 16 ? 1.f : i < 32 ? e1 : i < 48 ? e1 * f2[col] : e1 * f2[col] * f3[col]);
  };
  if constexpr (kFast) delta_chunk_solve_tc(p, As, beta, Bs, base, first, n, head, key);   // (the keys scaled to their block's end have been used)
  else delta_chunk_solve<T>(p, As, beta, base, first, n, head, key);
}

// One decay per head: the factor of a pair (i, s) is one number, exp(B_i - B_s) <= 1, so the sums over pairs are plain products q k^T and k k^T
// scaled afterwards (bfloat16 runs: m16n8k8 TF32 products of hi + lo operands, as in the scan; float32 runs: 32-bit multiply-adds).
template <typename T>
__global__ void __launch_bounds__(kDpThreads) delta_chunk_prep_head_kernel(const pcs_delta_chunk_params p) {
  extern __shared__ __align__(16) float sm[];
  const int D = p.dim, H = p.heads, D8 = (D + 7) & ~7, DP = ((D8 + 31) & ~31) + 4, U = 2 * p.kv_heads * D, L = (D + 63) & ~63;   // (rows 4 banks apart)
  float* qs = sm;              // [64][DP]
  float* ks = qs + kC * DP;    // [64][DP]
  float* As = ks + kC * DP;    // [64][64] beta_i A[i, s]
  float* beta = As + kC * kC;  // [64] each: step sizes, running sums of the log decays, their exponentials, the exponentials of what is left to the end
  float* Bs = beta + kC;
  float* eB = Bs + kC;
  float* eE = eB + kC;
  float* inv = eE + kC;        // [64][kTi] (bfloat16 runs)
  const int cn = blockIdx.x, head = blockIdx.y, hk = head / (H / p.kv_heads), tid = threadIdx.x;
  const int first = p.chunk_first[cn], n = p.chunk_len[cn];
  const long long base = static_cast<long long>(cn) * H + head;
  constexpr bool kFast = sizeof(T) == 2;
  constexpr float kLog = kFast ? 1.4426950408889634f : 1.f;
  auto ex = [](float x) { return kFast ? ex2(x) : expf(x); };
  const int warp = tid >> 5, lane = tid & 31;
  constexpr int kWarps = kDpThreads / 32;
  const float* qb = p.qk + hk * D;
  const float* kb = p.qk + (p.kv_heads + hk) * D;
  const bool vec = D % 4 == 0 && (reinterpret_cast<uintptr_t>(p.qk) & 15) == 0;
  if (vec) {
    for (int e = tid; e < 2 * kC * (D8 / 4); e += kDpThreads) {
      const int row = e / (D8 / 4), c = (e - row * (D8 / 4)) * 4, i = row & (kC - 1);
      float* dst = (row < kC ? qs : ks) + i * DP + c;
      if (i < n && c < D) cp_async16(dst, (row < kC ? qb : kb) + static_cast<long long>(first + i) * U + c);
      else *reinterpret_cast<float4*>(dst) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else {
    for (int e = tid; e < 2 * kC * D8; e += kDpThreads) {
      const int row = e / D8, c = e - row * D8, i = row & (kC - 1);
      (row < kC ? qs : ks)[i * DP + c] = i < n && c < D ? (row < kC ? qb : kb)[static_cast<long long>(first + i) * U + c] : 0.f;
    }
  }
  cp_async_commit();
  if (warp == 0) {   // lane owns tokens 2 lane and 2 lane + 1; tokens past the chunk's end decay nothing and write nothing
    float l[2];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int i = 2 * lane + x;
      l[x] = 0.f;
      float bt = 0.f;
      if (i < n) {
        const long long t = first + i;
        l[x] = kLog * head_log_decay(ldf(static_cast<const T*>(p.dec_a) + t * p.dec_stride + head) + p.dt_bias[head], p.rate[head]);
        bt = sigmoidf_(ldf(static_cast<const T*>(p.b) + t * p.b_stride + head));
      }
      beta[i] = bt;
    }
    float run = l[0] + l[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += up;
    }
    const float end = __shfl_sync(0xffffffffu, run, 31), b1 = run, b0 = run - l[1];
    Bs[2 * lane] = b0;
    Bs[2 * lane + 1] = b1;
    eB[2 * lane] = ex(b0);
    eB[2 * lane + 1] = ex(b1);
    eE[2 * lane] = ex(fminf(end - b0, 0.f));
    eE[2 * lane + 1] = ex(fminf(end - b1, 0.f));
  }
  float* ag = p.a + base * kC * kC;
  for (int e = tid; e < kC * kC; e += kDpThreads)
    if ((e & 63) > (e >> 6)) { ag[e] = 0.f; As[e] = 0.f; }   // above the diagonal
  cp_async_wait<0>();
  __syncthreads();
  auto put = [&](int i, int s, float qk, float kk) {
    if (s > i) return;
    const float f = ex(fminf(Bs[i] - Bs[s], 0.f));
    ag[i * kC + s] = qk * f;
    As[i * kC + s] = s < i ? beta[i] * kk * f : 0.f;
  };
  if (kFast) {
    const int g = lane >> 2, t = lane & 3;
    // ten tiles of 16 x 16 pairs on and below the diagonal, a warp each: (mi, nj) with nj <= mi
    for (int job = warp; job < 10; job += kWarps) {
      const int mi = job < 1 ? 0 : job < 3 ? 1 : job < 6 ? 2 : 3, nj = job - mi * (mi + 1) / 2;
      float q[3][2][4], k[3][2][4];
#pragma unroll
      for (int a = 0; a < 3; ++a)
#pragma unroll
        for (int u = 0; u < 2; ++u)
#pragma unroll
          for (int x = 0; x < 4; ++x) q[a][u][x] = k[a][u][x] = 0.f;
      const float* qa = qs + (16 * mi + g) * DP + t;
      const float* ka = ks + (16 * mi + g) * DP + t;
      const float* kn = ks + (16 * nj + g) * DP + t;
#pragma unroll 2
      for (int d = 0; d < D8; d += 8) {
        uint32_t ah[4], al[4], bh[2][2], bl[2][2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          split_tf32(kn[8 * u * DP + d], bh[u][0], bl[u][0]);
          split_tf32(kn[8 * u * DP + d + 4], bh[u][1], bl[u][1]);
        }
        split_tf32(qa[d], ah[0], al[0]);
        split_tf32(qa[d + 8 * DP], ah[1], al[1]);
        split_tf32(qa[d + 4], ah[2], al[2]);
        split_tf32(qa[d + 8 * DP + 4], ah[3], al[3]);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          mma_tf32(q[0][u], ah, bh[u][0], bh[u][1]);
          mma_tf32(q[1][u], ah, bl[u][0], bl[u][1]);
          mma_tf32(q[2][u], al, bh[u][0], bh[u][1]);
        }
        split_tf32(ka[d], ah[0], al[0]);
        split_tf32(ka[d + 8 * DP], ah[1], al[1]);
        split_tf32(ka[d + 4], ah[2], al[2]);
        split_tf32(ka[d + 8 * DP + 4], ah[3], al[3]);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          mma_tf32(k[0][u], ah, bh[u][0], bh[u][1]);
          mma_tf32(k[1][u], ah, bl[u][0], bl[u][1]);
          mma_tf32(k[2][u], al, bh[u][0], bh[u][1]);
        }
      }
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int x = 0; x < 4; ++x)
          put(16 * mi + g + 8 * (x >> 1), 16 * nj + 8 * u + 2 * t + (x & 1), q[0][u][x] + (q[1][u][x] + q[2][u][x]), k[0][u][x] + (k[1][u][x] + k[2][u][x]));
    }
  } else {
    for (int e = tid; e < (kC / 2) * (kC / 2 + 1) / 2; e += kDpThreads) {   // 2 x 2 pairs on and below the diagonal
      int bi = static_cast<int>((sqrtf(8.f * e + 1.f) - 1.f) * 0.5f);
      while ((bi + 1) * (bi + 2) / 2 <= e) ++bi;
      while (bi * (bi + 1) / 2 > e) --bi;
      const int i = 2 * bi, s = 2 * (e - bi * (bi + 1) / 2);
      float q[2][2] = {}, k[2][2] = {};
      for (int d = 0; d < D8; ++d) {
        const float s0 = ks[s * DP + d], s1 = ks[(s + 1) * DP + d];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const float qv = qs[(i + x) * DP + d], kv = ks[(i + x) * DP + d];
          q[x][0] = fmaf(qv, s0, q[x][0]);
          q[x][1] = fmaf(qv, s1, q[x][1]);
          k[x][0] = fmaf(kv, s0, k[x][0]);
          k[x][1] = fmaf(kv, s1, k[x][1]);
        }
      }
#pragma unroll
      for (int x = 0; x < 4; ++x) put(i + (x >> 1), s + (x & 1), q[x >> 1][x & 1], k[x >> 1][x & 1]);
    }
  }
  // what leaves the chunk
  {
    float* qd = p.qd + base * kC * D;
    float* kd = p.kd + base * kC * L;
    if (kFast) {   // the outgoing keys as fragments: a warp takes (16 channels, 8 tokens) at a time and writes 512 bytes
      for (int f = warp; f < (L / 16) * (kC / 8); f += kWarps) {
        const int mt = f >> 3, kt = f & 7;
        float o[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          const int i = kt * 8 + (lane & 3) + 4 * (r >> 1), d = mt * 16 + (lane >> 2) + 8 * (r & 1);
          o[r] = d < D ? ks[i * DP + d] * eE[i] : 0.f;
        }
        *reinterpret_cast<float4*>(kd + (static_cast<long long>(f) * 32 + lane) * 4) = make_float4(o[0], o[1], o[2], o[3]);
      }
    } else {
      for (int e = tid; e < kC * L; e += kDpThreads) {
        const int i = e / L, d = e - i * L;
        kd[static_cast<long long>(i) * L + delta_kd_slot(d)] = d < D ? ks[i * DP + d] * eE[i] : 0.f;
      }
    }
    for (int i = warp; i < kC; i += kWarps)
      for (int d = lane; d < D; d += 32) qd[i * D + d] = qs[i * DP + d] * eB[i];
    for (int d = tid; d < D; d += kDpThreads) p.g[base * D + d] = eB[kC - 1];
  }
  __syncthreads();
  auto key = [&](int i, int col) { return ks[i * DP + col] * eB[i]; };
  if constexpr (kFast) delta_chunk_solve_tc(p, As, beta, inv, base, first, n, head, key);
  else delta_chunk_solve<T>(p, As, beta, base, first, n, head, key);
}

// Block = (VS value columns, head, entry), 16 warps.  Both products split their sum over the warps and meet in `red`: u = u0 - w S over the
// channels, kd^T u over the tokens; a lane owns two rows, r and r + 16 of its warp's half of 64 (neighbours in
// the layouts the preparation writes), and half of the columns.  With NB = 2 the next chunk's w and kd travel under the whole of this chunk; with NB = 1 (wide heads) kd travels under
// the first product and the next chunk's w under the second.
constexpr int kDcThreads = 512;

template <int VS, int NB>
__global__ void __launch_bounds__(kDcThreads) delta_chunk_scan_kernel(const pcs_delta_chunk_params p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int CW = VS / 2;        // columns of a lane
  constexpr int LV = VS == 8 ? 3 : 4;
  const int D = p.dim, V = p.vdim, H = p.heads, L = (D + 63) & ~63, NT = L / 64, D8 = (D + 7) & ~7;
  float* ws = sm;                        // [NB][D][64]
  float* kds = ws + NB * D * kC;         // [NB][64][L]
  float* S = kds + NB * kC * L;          // [L][VS]
  float* us = S + L * VS;                // [64][VS]
  float* red = us + kC * VS;             // [8][64][VS]
  const int v0 = blockIdx.x * VS, head = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r = lane & 15, c4 = (lane >> 4) * CW, half = warp & 1, kp = warp >> 1;   // rows half * 32 + {r, r + 16} of 64; one of 8 parts of the sum
  const int n_chunks = p.seq_chunks[b];
  if (n_chunks <= 0) return;
  const long long c0 = p.seq_chunk0[b];
  const int vs = min(VS, V - v0);
  float* Sg = p.s_pool + (static_cast<long long>(p.seq_slot[b]) * H + head) * D * V;
  const bool fresh = p.seq_pos0[b] == 0;
  auto load_w = [&](int c) {
    const float* src = p.w + ((c0 + c) * H + head) * D8 * kC;
    float* dst = ws + (NB == 2 ? (c & 1) * D * kC : 0);
    for (int e = tid; e < D * (kC / 4); e += kDcThreads) cp_async16(dst + e * 4, src + e * 4);
  };
  auto load_kd = [&](int c) {
    const float* src = p.kd + ((c0 + c) * H + head) * kC * L;
    float* dst = kds + (NB == 2 ? (c & 1) * kC * L : 0);
    for (int e = tid; e < kC * (L / 4); e += kDcThreads) cp_async16(dst + e * 4, src + e * 4);
  };
  load_w(0);
  cp_async_commit();
  load_kd(0);
  cp_async_commit();
  for (int e = tid; e < L * VS; e += kDcThreads) {
    const int d = e >> LV, c = e & (VS - 1);
    S[e] = (!fresh && d < D && c < vs) ? Sg[static_cast<long long>(d) * V + v0 + c] : 0.f;
  }
  // phase 1: warp pair -> channels [d_lo, d_hi); phase 2: warp pair -> (64-channel tile, part of the tokens)
  const int dw = (D + 7) / 8, d_lo = min(D, kp * dw), d_hi = min(D, d_lo + dw);
  const int parts = 8 / NT, tile = kp % NT, part = kp / NT, tw = kC / parts;
  const int i_lo = part * tw;
  const bool busy2 = part < parts;
  constexpr int kOut1 = kC * VS / kDcThreads;        // outputs of phase 1 per thread
  constexpr int kOut2 = 256 * VS / kDcThreads;       // of phase 2, at most (dim 256)
  float u0[kOut1], gd[kOut2];   // this chunk's right-hand sides and decays; the next chunk's are requested a chunk ahead
  auto load_u = [&](int c, float (&o)[kOut1]) {
    const float* src = p.u + ((c0 + c) * H + head) * kC * V + v0;
#pragma unroll
    for (int m = 0; m < kOut1; ++m) {
      const int e = tid + m * kDcThreads;
      o[m] = (e & (VS - 1)) < vs ? src[static_cast<long long>(e >> LV) * V + (e & (VS - 1))] : 0.f;
    }
  };
  auto load_g = [&](int c, float (&o)[kOut2]) {
    const float* src = p.g + ((c0 + c) * H + head) * D;
#pragma unroll
    for (int m = 0; m < kOut2; ++m) {
      const int d = (tid + m * kDcThreads) >> LV;
      o[m] = d < D ? src[d] : 0.f;
    }
  };
  load_u(0, u0);
  load_g(0, gd);
  for (int c = 0; c < n_chunks; ++c) {
    const long long base = (c0 + c) * H + head;
    float* ug = p.u + base * kC * V + v0;
    float un[kOut1], gn[kOut2];
    if (c + 1 < n_chunks) {
      load_u(c + 1, un);
      load_g(c + 1, gn);
    }
    cp_async_wait<1>();
    __syncthreads();   // w of this chunk, and the state; the buffers of the chunk before are free
    if (NB == 2) {
      if (c + 1 < n_chunks) load_w(c + 1);
      cp_async_commit();
      if (c + 1 < n_chunks) load_kd(c + 1);
      cp_async_commit();
    }
    {
      const float* wc = ws + (NB == 2 ? (c & 1) * D * kC : 0);
      float acc[2][CW];
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int y = 0; y < CW; ++y) acc[x][y] = 0.f;
#pragma unroll 8
      for (int d = d_lo; d < d_hi; ++d) {
        const float2 w2 = *reinterpret_cast<const float2*>(wc + d * kC + 4 * r + 2 * half);
        const float wv[2] = {w2.x, w2.y};
#pragma unroll
        for (int y = 0; y < CW; y += 4) {
          const float4 s4 = *reinterpret_cast<const float4*>(S + d * VS + c4 + y);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            acc[x][y] = fmaf(wv[x], s4.x, acc[x][y]);
            acc[x][y + 1] = fmaf(wv[x], s4.y, acc[x][y + 1]);
            acc[x][y + 2] = fmaf(wv[x], s4.z, acc[x][y + 2]);
            acc[x][y + 3] = fmaf(wv[x], s4.w, acc[x][y + 3]);
          }
        }
      }
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int y = 0; y < CW; y += 4)
          *reinterpret_cast<float4*>(red + kp * (kC * VS) + (half * 32 + r + 16 * x) * VS + c4 + y) = make_float4(acc[x][y], acc[x][y + 1], acc[x][y + 2], acc[x][y + 3]);
    }
    __syncthreads();
    if (NB == 1) {
      if (c + 1 < n_chunks) load_w(c + 1);
      cp_async_commit();
    }
#pragma unroll
    for (int m = 0; m < kOut1; ++m) {
      const int e = tid + m * kDcThreads;
      float a = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) a += red[w * (kC * VS) + e];
      const float u = u0[m] - a;
      us[e] = u;
      if ((e & (VS - 1)) < vs) ug[static_cast<long long>(e >> LV) * V + (e & (VS - 1))] = u;
    }
    cp_async_wait<NB>();
    __syncthreads();   // kd of this chunk, and u; `red` is free again
    if (busy2) {
      const float* kc = kds + (NB == 2 ? (c & 1) * kC * L : 0);
      float acc[2][CW];
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int y = 0; y < CW; ++y) acc[x][y] = 0.f;
#pragma unroll 8
      for (int i = i_lo; i < i_lo + tw; ++i) {
        const float2 k2 = *reinterpret_cast<const float2*>(kc + i * L + tile * 64 + 4 * r + 2 * half);
        const float kv[2] = {k2.x, k2.y};
#pragma unroll
        for (int y = 0; y < CW; y += 4) {
          const float4 u4 = *reinterpret_cast<const float4*>(us + i * VS + c4 + y);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            acc[x][y] = fmaf(kv[x], u4.x, acc[x][y]);
            acc[x][y + 1] = fmaf(kv[x], u4.y, acc[x][y + 1]);
            acc[x][y + 2] = fmaf(kv[x], u4.z, acc[x][y + 2]);
            acc[x][y + 3] = fmaf(kv[x], u4.w, acc[x][y + 3]);
          }
        }
      }
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int y = 0; y < CW; y += 4)
          *reinterpret_cast<float4*>(red + part * (L * VS) + (tile * 64 + half * 32 + r + 16 * x) * VS + c4 + y) = make_float4(acc[x][y], acc[x][y + 1], acc[x][y + 2], acc[x][y + 3]);
    }
    __syncthreads();
    if (NB == 1) {
      if (c + 1 < n_chunks) load_kd(c + 1);
      cp_async_commit();
    }
    float* sg = p.s + base * D * V + v0;
#pragma unroll
    for (int m = 0; m < kOut2; ++m) {
      const int e = tid + m * kDcThreads;
      if (e < L * VS) {
        float a = 0.f;
        for (int w = 0; w < parts; ++w) a += red[w * (L * VS) + e];
        const int d = e >> LV, cc = e & (VS - 1);
        const float old = S[e];
        if (d < D && cc < vs) sg[static_cast<long long>(d) * V + cc] = old;
        S[e] = fmaf(gd[m], old, a);
      }
      gd[m] = gn[m];
    }
#pragma unroll
    for (int m = 0; m < kOut1; ++m) u0[m] = un[m];
  }
  cp_async_wait<0>();
  __syncthreads();
  for (int e = tid; e < D * VS; e += kDcThreads)
    if ((e & (VS - 1)) < vs) Sg[static_cast<long long>(e >> LV) * V + v0 + (e & (VS - 1))] = S[e];
}

// The same in bfloat16 runs, the two products on the tensor cores: m16n8k8 with every 32-bit operand split into two TF32 parts, x = hi + lo, and
// the three products hi hi + hi lo + lo hi in 32-bit accumulators (what is dropped is 2^-22 of a product; states stay 32-bit).  Block = (8 NV
// value columns, head, entry), 8 warps.  The preparation writes w and kd as fragments, so an operand tile is one 16-byte load per lane.
//   u = u0 - w S      warp = (16 tokens, half of the channels); the two halves meet in shared memory
//   S = g S + kd^T u  warp = 16 channels (and 16 more at dim > 128): no sum leaves the warp, S stays in its accumulators
// S and u also sit in shared memory as [row][8] tiles: a B fragment is 32 neighbouring numbers.
constexpr int kDtThreads = 256;

template <int NV, int NB, int MT>   // MT: 16-channel tiles per warp (dim <= 128 MT)
__global__ void __launch_bounds__(kDtThreads) delta_chunk_scan_tc_kernel(const pcs_delta_chunk_params p) {
  extern __shared__ __align__(16) float sm[];
  constexpr int VS = 8 * NV;
  const int D = p.dim, V = p.vdim, H = p.heads, L = (D + 63) & ~63, D8 = (D + 7) & ~7, KT = D8 / 8;
  float* ws = sm;                        // [NB][D8 / 8][4][32][4]
  float* kds = ws + NB * D8 * kC;        // [NB][L / 16][8][32][4]
  float* S = kds + NB * kC * L;          // [NV][128 MT][8]
  float* us = S + NV * 128 * MT * 8;     // [NV][64][8]
  float* red = us + NV * kC * 8;         // [NV][64][8]
  const int v0 = blockIdx.x * VS, head = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3;
  const int n_chunks = p.seq_chunks[b];
  if (n_chunks <= 0) return;
  const long long c0 = p.seq_chunk0[b];
  float* Sg = p.s_pool + (static_cast<long long>(p.seq_slot[b]) * H + head) * D * V;
  const bool fresh = p.seq_pos0[b] == 0;
  auto load_w = [&](int c) {
    const float* src = p.w + ((c0 + c) * H + head) * D8 * kC;
    float* dst = ws + (NB == 2 ? (c & 1) * D8 * kC : 0);
    for (int e = tid; e < D8 * (kC / 4); e += kDtThreads) cp_async16(dst + e * 4, src + e * 4);
  };
  auto load_kd = [&](int c) {
    const float* src = p.kd + ((c0 + c) * H + head) * kC * L;
    float* dst = kds + (NB == 2 ? (c & 1) * kC * L : 0);
    for (int e = tid; e < kC * (L / 4); e += kDtThreads) cp_async16(dst + e * 4, src + e * 4);
  };
  load_w(0);
  cp_async_commit();
  load_kd(0);
  cp_async_commit();
  // this thread's state: rows 16 (warp + 8 m) + g (+ 8), columns 8 n + 2 t (+ 1)
  float st[MT][NV][4];
  const bool even = (V & 1) == 0;
  auto load2 = [&](const float* row, int col, float& x, float& y) {   // two neighbouring columns of a row, those past vdim zero
    if (even) {
      const float2 q = col < V ? *reinterpret_cast<const float2*>(row + col) : make_float2(0.f, 0.f);
      x = q.x;
      y = q.y;
    } else {
      x = col < V ? row[col] : 0.f;
      y = col + 1 < V ? row[col + 1] : 0.f;
    }
  };
  auto store2 = [&](float* row, int col, float x, float y) {
    if (even) {
      if (col < V) *reinterpret_cast<float2*>(row + col) = make_float2(x, y);
    } else {
      if (col < V) row[col] = x;
      if (col + 1 < V) row[col + 1] = y;
    }
  };
  auto publish = [&]() {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < NV; ++n) {
        float* o = S + (n * 128 * MT + 16 * (warp + 8 * m) + g) * 8 + 2 * t;
        *reinterpret_cast<float2*>(o) = make_float2(st[m][n][0], st[m][n][1]);
        *reinterpret_cast<float2*>(o + 64) = make_float2(st[m][n][2], st[m][n][3]);
      }
  };
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = 16 * (warp + 8 * m) + g + 8 * h;
        st[m][n][2 * h] = st[m][n][2 * h + 1] = 0.f;
        if (!fresh && d < D) load2(Sg + static_cast<long long>(d) * V, v0 + 8 * n + 2 * t, st[m][n][2 * h], st[m][n][2 * h + 1]);
      }
  publish();
  const int mi = warp & 3, kh = warp >> 2, kt_lo = kh ? (KT + 1) / 2 : 0, kt_hi = kh ? KT : (KT + 1) / 2;
  float u0[NV][4], gd[MT][2], un[NV][4], gn[MT][2];
  auto load_u = [&](int c, float (&o)[NV][4]) {
    if (kh != 0) return;
    const float* src = p.u + ((c0 + c) * H + head) * kC * V;
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) load2(src + static_cast<long long>(16 * mi + g + 8 * h) * V, v0 + 8 * n + 2 * t, o[n][2 * h], o[n][2 * h + 1]);
  };
  auto load_g = [&](int c, float (&o)[MT][2]) {
    const float* src = p.g + ((c0 + c) * H + head) * D;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = 16 * (warp + 8 * m) + g + 8 * h;
        o[m][h] = d < D ? src[d] : 0.f;
      }
  };
  load_u(0, u0);
  load_g(0, gd);
  // one k-step: the A fragment against every column tile; three accumulators per tile, so that a chain is one product per step
  auto step = [&](const float* af, const float* bt, int b_tile, float (&hh)[NV][4], float (&hl)[NV][4], float (&lh)[NV][4]) {
    const float4 a4 = *reinterpret_cast<const float4*>(af + lane * 4);
    uint32_t ah[4], al[4];
    split_tf32(a4.x, ah[0], al[0]);
    split_tf32(a4.y, ah[1], al[1]);
    split_tf32(a4.z, ah[2], al[2]);
    split_tf32(a4.w, ah[3], al[3]);
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      uint32_t h0, l0, h1, l1;
      split_tf32(bt[n * b_tile + t * 8 + g], h0, l0);
      split_tf32(bt[n * b_tile + 32 + t * 8 + g], h1, l1);
      mma_tf32(hh[n], ah, h0, h1);
      mma_tf32(hl[n], ah, l0, l1);
      mma_tf32(lh[n], al, h0, h1);
    }
  };
  for (int c = 0; c < n_chunks; ++c) {
    const long long base = (c0 + c) * H + head;
    if (c + 1 < n_chunks) {
      load_u(c + 1, un);
      load_g(c + 1, gn);
    }
    cp_async_wait<1>();
    __syncthreads();   // w of this chunk, and the state; the buffers of the chunk before are free
    if (NB == 2) {
      if (c + 1 < n_chunks) load_w(c + 1);
      cp_async_commit();
      if (c + 1 < n_chunks) load_kd(c + 1);
      cp_async_commit();
    }
    float hh[NV][4], hl[NV][4], lh[NV][4];
    auto zero = [&](float (&x)[NV][4]) {
#pragma unroll
      for (int n = 0; n < NV; ++n) x[n][0] = x[n][1] = x[n][2] = x[n][3] = 0.f;
    };
    zero(hh);
    zero(hl);
    zero(lh);
    {
      const float* wc = ws + (NB == 2 ? (c & 1) * D8 * kC : 0) + mi * 128;
#pragma unroll 4
      for (int kt = kt_lo; kt < kt_hi; ++kt) step(wc + kt * 512, S + kt * 64, 128 * MT * 8, hh, hl, lh);
    }
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) hh[n][x] += hl[n][x] + lh[n][x];
    if (kh == 1) {
#pragma unroll
      for (int n = 0; n < NV; ++n) {
        float* o = red + (n * kC + 16 * mi + g) * 8 + 2 * t;
        *reinterpret_cast<float2*>(o) = make_float2(hh[n][0], hh[n][1]);
        *reinterpret_cast<float2*>(o + 64) = make_float2(hh[n][2], hh[n][3]);
      }
    }
    __syncthreads();
    if (NB == 1) {
      if (c + 1 < n_chunks) load_w(c + 1);
      cp_async_commit();
    }
    if (kh == 0) {
      float* ug = p.u + base * kC * V;
#pragma unroll
      for (int n = 0; n < NV; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int i = 16 * mi + g + 8 * h, o = (n * kC + i) * 8 + 2 * t;
          const float2 r2 = *reinterpret_cast<const float2*>(red + o);
          const float x = u0[n][2 * h] - (hh[n][2 * h] + r2.x), y = u0[n][2 * h + 1] - (hh[n][2 * h + 1] + r2.y);
          *reinterpret_cast<float2*>(us + o) = make_float2(x, y);
          store2(ug + static_cast<long long>(i) * V, v0 + 8 * n + 2 * t, x, y);
        }
    }
    cp_async_wait<NB>();
    __syncthreads();   // kd of this chunk, and u
    float* sg = p.s + base * D * V;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int mt = warp + 8 * m;
      if (16 * mt < D) {
#pragma unroll
        for (int n = 0; n < NV; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int d = 16 * mt + g + 8 * h;
            if (d < D) store2(sg + static_cast<long long>(d) * V, v0 + 8 * n + 2 * t, st[m][n][2 * h], st[m][n][2 * h + 1]);   // the state this chunk starts from
          }
        zero(hh);
        zero(hl);
        zero(lh);
        const float* kc = kds + (NB == 2 ? (c & 1) * kC * L : 0) + mt * 1024;
#pragma unroll
        for (int kt = 0; kt < 8; ++kt) step(kc + kt * 128, us + kt * 64, kC * 8, hh, hl, lh);
#pragma unroll
        for (int n = 0; n < NV; ++n)
#pragma unroll
          for (int x = 0; x < 4; ++x) st[m][n][x] = fmaf(gd[m][x >> 1], st[m][n][x], hh[n][x] + (hl[n][x] + lh[n][x]));
      }
#pragma unroll
      for (int h = 0; h < 2; ++h) gd[m][h] = gn[m][h];
    }
    publish();
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) u0[n][x] = un[n][x];
    if (NB == 1) {
      __syncthreads();   // every warp has read this chunk's kd
      if (c + 1 < n_chunks) load_kd(c + 1);
      cp_async_commit();
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NV; ++n)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = 16 * (warp + 8 * m) + g + 8 * h;
        if (d < D) store2(Sg + static_cast<long long>(d) * V, v0 + 8 * n + 2 * t, st[m][n][2 * h], st[m][n][2 * h + 1]);
      }
}

template <int NV, int NB, int MT>
static int launch_delta_chunk_scan_tc(const pcs_delta_chunk_params& p, size_t smem, cudaStream_t st) {
  PCS_CHECK_CUDA(cudaFuncSetAttribute(delta_chunk_scan_tc_kernel<NV, NB, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
  delta_chunk_scan_tc_kernel<NV, NB, MT><<<dim3((p.vdim + 8 * NV - 1) / (8 * NV), p.heads, p.n_seqs), kDtThreads, smem, st>>>(p);
  PCS_CHECK_CUDA(cudaGetLastError());
  count_launch();
  return PCS_OK;
}

template <int MT>
static int launch_delta_chunk_scan_tc(const pcs_delta_chunk_params& p, cudaStream_t st) {
  const int L = (p.dim + 63) & ~63, D8 = (p.dim + 7) & ~7;
  auto smem = [&](int nv, int nb) { return (static_cast<size_t>(nb) * kC * (D8 + L) + static_cast<size_t>(nv) * 8 * (128 * MT + 2 * kC)) * sizeof(float); };
  // 8 columns per block where that still is one block per SM, else 16 (half of the chunk traffic); two buffers where they fit
  const long long rows = static_cast<long long>(p.heads) * p.n_seqs;
  const int nv = rows * ((p.vdim + 7) / 8) <= 148 ? 1 : 2;
  const bool one_wave = rows * ((p.vdim + 8 * nv - 1) / (8 * nv)) <= 148;
  const bool two = smem(nv, 2) <= (one_wave ? 227u : 112u) * 1024u;
  if (nv == 1) return two ? launch_delta_chunk_scan_tc<1, 2, MT>(p, smem(1, 2), st) : launch_delta_chunk_scan_tc<1, 1, MT>(p, smem(1, 1), st);
  return two ? launch_delta_chunk_scan_tc<2, 2, MT>(p, smem(2, 2), st) : launch_delta_chunk_scan_tc<2, 1, MT>(p, smem(2, 1), st);
}

template <int VS, int NB>
static int launch_delta_chunk_scan(const pcs_delta_chunk_params& p, size_t smem, cudaStream_t st) {
  PCS_CHECK_CUDA(cudaFuncSetAttribute(delta_chunk_scan_kernel<VS, NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
  delta_chunk_scan_kernel<VS, NB><<<dim3((p.vdim + VS - 1) / VS, p.heads, p.n_seqs), kDcThreads, smem, st>>>(p);
  PCS_CHECK_CUDA(cudaGetLastError());
  count_launch();
  return PCS_OK;
}

// ---- read-out of the chunks (bfloat16 runs) ---------------------------------------------------------------------------------------
// Block = (chunk, head), a warp = 32 value columns: o = qd S + a u over dim + 64 terms, then the head's norm and gate on the accumulators, and the
// result's rows.  The result leaves in bfloat16, so the operands enter as hi + lo bfloat16 pairs (hi hi + hi lo + lo hi in 32-bit accumulators,
// about 2^-16 of a product); the state itself stays as it is.  [qd | a] is staged in shared memory as such pairs, S and u are read once, a step ahead.
constexpr int kDoMaxWarps = 16;

__global__ void __launch_bounds__(kDoMaxWarps * 32) delta_chunk_out_kernel(const pcs_delta_chunk_params p, const pcs_headnorm_params o) {
  extern __shared__ __align__(16) float sm[];
  const int D = p.dim, V = p.vdim, H = p.heads, D16 = (D + 15) & ~15, LD = D16 + kC + 8;   // (rows an odd number of 16-byte pieces apart)
  __nv_bfloat16* Ah = reinterpret_cast<__nv_bfloat16*>(sm);   // [64][LD]
  __nv_bfloat16* Al = Ah + kC * LD;                           // [64][LD]
  float* red = reinterpret_cast<float*>(Al + kC * LD);        // [warps][64], then [64]
  const int cn = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, nthr = blockDim.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const long long base = static_cast<long long>(cn) * H + head;
  const int first = p.chunk_first[cn], n = p.chunk_len[cn];
  const float* qd = p.qd + base * kC * D;
  const float* ag = p.a + base * kC * kC;
  auto put = [&](int i, int c, const float (&x)[4]) {
    uint2 hi, lo;
    hi.x = split_pair(x[0], x[1], lo.x);
    hi.y = split_pair(x[2], x[3], lo.y);
    *reinterpret_cast<uint2*>(Ah + i * LD + c) = hi;
    *reinterpret_cast<uint2*>(Al + i * LD + c) = lo;
  };
  // (place x of the warp's tile q is its column 4 x + q: a lane's four values of a row are neighbours)
  const int c0 = warp * 32 + 4 * g, KD = D16 / 16, KT = KD + kC / 16;
  const float* sg = p.s + base * D * V;
  const float* ug = p.u + base * kC * V;
  const bool quads = V % 4 == 0;
  auto load = [&](int kt, float (&b)[4][4]) {   // rows 2t, 2t + 1, 2t + 8, 2t + 9 of the step's 16
    const bool state = kt < KD;
    const int r0 = 16 * (state ? kt : kt - KD) + 2 * t;
    const float* src = (state ? sg : ug) + static_cast<long long>(r0) * V + c0;
#pragma unroll
    for (int h = 0; h < 4; ++h) {
      const int dr = (h & 1) + 8 * (h >> 1);
      const bool ok = kt < KT && (!state || r0 + dr < D);
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      const float* r = src + static_cast<long long>(dr) * V;
      if (ok && quads) {
        if (c0 < V) x = *reinterpret_cast<const float4*>(r);
      } else if (ok) {
        if (c0 < V) x.x = r[0];
        if (c0 + 1 < V) x.y = r[1];
        if (c0 + 2 < V) x.z = r[2];
        if (c0 + 3 < V) x.w = r[3];
      }
      b[0][h] = x.x;
      b[1][h] = x.y;
      b[2][h] = x.z;
      b[3][h] = x.w;
    }
  };
  float acc[4][4][4], nx[4][4];
#pragma unroll
  for (int q = 0; q < 4; ++q)
#pragma unroll
    for (int m = 0; m < 4; ++m) acc[q][m][0] = acc[q][m][1] = acc[q][m][2] = acc[q][m][3] = 0.f;
  load(0, nx);
  const int per = D16 / 4, pieces = kC * (per + kC / 4);   // a row's pieces of qd, then of a
  for (int e0 = tid; e0 < pieces; e0 += 4 * nthr) {        // (four requests before the first is used)
    float x[4][4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int e = e0 + k * nthr;
      x[k][0] = x[k][1] = x[k][2] = x[k][3] = 0.f;
      if (e < pieces) {
        const int i = e / (per + kC / 4), c = e - i * (per + kC / 4);
        if (c >= per) {
          ldx(ag + i * kC + (c - per) * 4, x[k]);
        } else if (D % 4 == 0) {
          if (4 * c < D) ldx(qd + i * D + 4 * c, x[k]);
        } else {
#pragma unroll
          for (int y = 0; y < 4; ++y)
            if (4 * c + y < D) x[k][y] = qd[i * D + 4 * c + y];
        }
      }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int e = e0 + k * nthr;
      if (e < pieces) {
        const int i = e / (per + kC / 4);
        put(i, 4 * (e - i * (per + kC / 4)), x[k]);
      }
    }
  }
  __syncthreads();
  const uint32_t a_hi = static_cast<uint32_t>(__cvta_generic_to_shared(Ah)) + ((lane & 15) * LD + (lane >> 4) * 8) * 2, a_lo = a_hi + kC * LD * 2;
#pragma unroll 1
  for (int kt = 0; kt < KT; ++kt) {
    uint32_t bh[4][2], bl[4][2];
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      bh[q][0] = split_pair(nx[q][0], nx[q][1], bl[q][0]);
      bh[q][1] = split_pair(nx[q][2], nx[q][3], bl[q][1]);
    }
    load(kt + 1, nx);
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      if (m < kt - KD) continue;   // `a` is zero above the diagonal
      uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
      ldsm_x4(a_hi + (m * 16 * LD + kt * 16) * 2, h0, h1, h2, h3);
      ldsm_x4(a_lo + (m * 16 * LD + kt * 16) * 2, l0, l1, l2, l3);
#pragma unroll
      for (int q = 0; q < 4; ++q) mma_bf16(acc[q][m], h0, h1, h2, h3, bh[q][0], bh[q][1]);
#pragma unroll
      for (int q = 0; q < 4; ++q) mma_bf16(acc[q][m], h0, h1, h2, h3, bl[q][0], bl[q][1]);
#pragma unroll
      for (int q = 0; q < 4; ++q) mma_bf16(acc[q][m], l0, l1, l2, l3, bh[q][0], bh[q][1]);
    }
  }
  // the head's mean square per token: a row's columns are spread over 4 lanes and all warps
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float ss = 0.f;
#pragma unroll
      for (int q = 0; q < 4; ++q) ss = fmaf(acc[q][m][2 * h], acc[q][m][2 * h], fmaf(acc[q][m][2 * h + 1], acc[q][m][2 * h + 1], ss));
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (t == 0) red[warp * kC + 16 * m + g + 8 * h] = ss;
    }
  __syncthreads();
  float inv = 0.f;
  for (int i = tid; i < kC; i += nthr) {   // (at least two warps)
    for (int w = 0; w < nthr / 32; ++w) inv += red[w * kC + i];
    inv = o.out_scale / sqrtf(inv / static_cast<float>(V) + o.eps);
  }
  __syncthreads();
  if (tid < kC) red[tid] = inv;
  __syncthreads();
  const __nv_bfloat16* gate = static_cast<const __nv_bfloat16*>(o.g) + static_cast<long long>(first) * o.g_stride + head * V;
  const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(o.w);
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(o.out) + static_cast<long long>(first) * o.out_stride + head * V;
  const bool vec = quads && o.out_stride % 4 == 0 && o.g_stride % 4 == 0 && ((reinterpret_cast<uintptr_t>(o.g) | reinterpret_cast<uintptr_t>(o.out) | reinterpret_cast<uintptr_t>(o.w)) & 7) == 0;
  auto unpack = [](const uint2& v, float (&f)[4]) {
    f[0] = __uint_as_float(v.x << 16);
    f[1] = __uint_as_float(v.x & 0xffff0000u);
    f[2] = __uint_as_float(v.y << 16);
    f[3] = __uint_as_float(v.y & 0xffff0000u);
  };
  auto gated = [&](float x, float f, float wv, float gv) { return x * f * wv * sigmoidf_(gv) * (o.silu ? gv : 1.f); };
#pragma unroll
  for (int e = 0; e < 2; ++e) {   // this lane's columns c .. c + 3 (places 2t + e), eight tokens: all gates are requested before the first result leaves
    const int c = warp * 32 + 4 * (2 * t + e);
    if (c >= V) continue;
    if (vec) {
      uint2 gv[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int i = 16 * (k >> 1) + g + 8 * (k & 1);
        gv[k] = i < n ? *reinterpret_cast<const uint2*>(gate + static_cast<long long>(i) * o.g_stride + c) : make_uint2(0u, 0u);
      }
      float wv[4];
      unpack(*reinterpret_cast<const uint2*>(w + c), wv);
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int m = k >> 1, x = 2 * (k & 1) + e, i = 16 * m + g + 8 * (k & 1);
        if (i >= n) continue;
        const float f = red[i];
        float gf[4];
        unpack(gv[k], gf);
        uint2 r;
        r.x = pack_bf16(gated(acc[0][m][x], f, wv[0], gf[0]), gated(acc[1][m][x], f, wv[1], gf[1]));
        r.y = pack_bf16(gated(acc[2][m][x], f, wv[2], gf[2]), gated(acc[3][m][x], f, wv[3], gf[3]));
        *reinterpret_cast<uint2*>(out + static_cast<long long>(i) * o.out_stride + c) = r;
      }
    } else {
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int m = k >> 1, x = 2 * (k & 1) + e, i = 16 * m + g + 8 * (k & 1);
        if (i >= n) continue;
        const float f = red[i];
#pragma unroll
        for (int q = 0; q < 4; ++q)
          if (c + q < V)
            stf(out + static_cast<long long>(i) * o.out_stride + c + q, gated(acc[q][m][x], f, ldf(w + c + q), ldf(gate + static_cast<long long>(i) * o.g_stride + c + q)));
      }
    }
  }
}

// ---- per-head norm and gate ------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const pcs_headnorm_params p) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, V = p.vdim, H = p.heads;
  const long long e = static_cast<long long>(blockIdx.x) * (blockDim.x >> 5) + warp;
  if (e >= static_cast<long long>(p.n_tokens) * H) return;
  const long long t = e / H;
  const int h = static_cast<int>(e - t * H);
  long long row = e;
  if (p.tok_row) {
    const int tr = p.tok_row[t];
    row = (static_cast<long long>(tr / p.chunk_size) * H + h) * p.chunk_size + tr % p.chunk_size;
  }
  const float* o = p.o + row * V;
  const T* g = static_cast<const T*>(p.g) + t * p.g_stride + h * V;
  const T* w = static_cast<const T*>(p.w);
  T* out = static_cast<T*>(p.out) + t * p.out_stride + h * V;
  constexpr int KEEP = 16;   // columns of a lane that stay in registers
  float ov[KEEP], gv[KEEP], wv[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int c = lane + u * 32;
    ov[u] = c < V ? o[c] : 0.f;
    gv[u] = c < V ? ldf(g + c) : 0.f;
    wv[u] = c < V ? ldf(w + c) : 0.f;
  }
#pragma unroll
  for (int u = 0; u < KEEP; ++u) ss = fmaf(ov[u], ov[u], ss);
  for (int c = lane + KEEP * 32; c < V; c += 32) ss = fmaf(o[c], o[c], ss);
  ss = warp_sum(ss);
  const float inv = p.out_scale / sqrtf(ss / static_cast<float>(V) + p.eps);
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int c = lane + u * 32;
    if (c < V) stf(out + c, ov[u] * inv * wv[u] * sigmoidf_(gv[u]) * (p.silu ? gv[u] : 1.f));
  }
  for (int c = lane + KEEP * 32; c < V; c += 32) {
    const float gc = ldf(g + c);
    stf(out + c, o[c] * inv * ldf(w + c) * sigmoidf_(gc) * (p.silu ? gc : 1.f));
  }
}

}  // namespace pcs

static int check_short_conv(const pcs_shortconv_params* p, const char* what, bool* vec) {
  PCS_REQUIRE(p->proj && p->conv_w && p->qk_out && p->v_out && p->tok_seq && p->tok_pos && p->seq_slot && p->seq_pos0 && p->seq_len && p->seq_par,
              "%s: null tensor", what);
  PCS_REQUIRE(p->kv_heads > 0 && p->dim > 0 && p->v_width > 0 && p->c_off >= 0 && p->taps >= 1 && p->taps <= pcs::kScMaxTaps && (p->tail || p->taps == 1),
              "%s: bad sizes (taps %d of at most %d)", what, p->taps, pcs::kScMaxTaps);
  const int piece = p->dtype == PCS_BF16 ? 8 : 4;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  *vec = p->impl != 1 && p->taps <= 4 && p->dim % piece == 0 && p->v_width % piece == 0 && p->c_off % piece == 0 && p->row_stride % piece == 0 &&
         p->dim <= 256 * piece && al(p->proj) && al(p->conv_w) && al(p->tail) && al(p->qk_out) && al(p->v_out);
  return PCS_OK;
}

PCS_API int pcs_short_conv(const pcs_shortconv_params* p, void* stream) {
  PCS_REQUIRE(p, "pcs_short_conv: null params");
  if (p->n_tokens == 0) return PCS_OK;
  bool vec = false;
  if (int rc = check_short_conv(p, "pcs_short_conv", &vec)) return rc;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  PCS_DISPATCH(p->dtype, return pcs::launch_short_conv<T>(*p, nullptr, st, vec));
}

PCS_API int pcs_delta_inputs(const pcs_shortconv_params* p, const pcs_lowrank_params* q, void* stream) {
  PCS_REQUIRE(p && q, "pcs_delta_inputs: null params");
  if (p->n_tokens == 0) return PCS_OK;
  bool vec = false;
  if (int rc = check_short_conv(p, "pcs_delta_inputs", &vec)) return rc;
  if (!vec) return pcs::set_error(PCS_ERR_UNSUPPORTED, "pcs_delta_inputs: sizes off the 16-byte pieces take pcs_short_conv and products of their own");
  PCS_REQUIRE(q->a2 && q->dt_bias && q->rate && q->decay_out && q->g2 && q->gate_out && q->heads > 0 && q->dim > 0 && q->decay_rank > 0 && q->gate_rank > 0 &&
                  q->gate_width > 0 && q->a_off >= 0 && q->g_off >= 0, "pcs_delta_inputs: bad low-rank products");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  PCS_DISPATCH(p->dtype, return pcs::launch_short_conv<T>(*p, q, st, true));
}

PCS_API int pcs_delta_scan(const pcs_delta_params* p, void* stream) {
  PCS_REQUIRE(p, "pcs_delta_scan: null params");
  if (p->n_seqs == 0 || p->n_tokens == 0) return PCS_OK;
  PCS_REQUIRE(p->qk && p->v && p->b && p->o && p->s_pool && p->seq_slot && p->seq_pos0 && p->seq_len && p->seq_off, "pcs_delta_scan: null tensor");
  PCS_REQUIRE(p->decay || (p->a && p->dt_bias && p->rate), "pcs_delta_scan: neither decays per channel nor what per-head decays are formed of");
  PCS_REQUIRE(p->heads > 0 && p->heads <= 65535 && p->kv_heads > 0 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->vdim > 0, "pcs_delta_scan: bad sizes");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool aligned = p->dim % 4 == 0 && ((reinterpret_cast<uintptr_t>(p->qk) | reinterpret_cast<uintptr_t>(p->decay)) & 15) == 0;
  if (p->impl != 1 && p->dim <= 256 && aligned) {
    // warps per block halve until the launch has two blocks per SM (or one warp is left)
    int W = 8;
    while (W > 1 && 8 * (W / 2) >= p->vdim) W /= 2;
    auto blocks = [&](int w) { return static_cast<long long>(p->n_seqs) * p->heads * ((p->vdim + 8 * w - 1) / (8 * w)); };
    while (W > 1 && blocks(W) < 2 * 148) W /= 2;
    dim3 grid(p->n_seqs, p->heads, (p->vdim + 8 * W - 1) / (8 * W));
#define PCS_DELTA_REG(MV) \
  PCS_DISPATCH(p->dtype, { \
    const size_t row = static_cast<size_t>(pcs::kDsRing) * 16 * MV * sizeof(float); \
    if (p->decay) pcs::delta_scan_reg_kernel<T, MV, false><<<grid, 32 * W, 3 * row, st>>>(*p, W); \
    else pcs::delta_scan_reg_kernel<T, MV, true><<<grid, 32 * W, 2 * row, st>>>(*p, W); \
  })
    if (p->dim <= 32) PCS_DELTA_REG(2);
    else if (p->dim <= 64) PCS_DELTA_REG(4);
    else if (p->dim <= 128) PCS_DELTA_REG(8);
    else PCS_DELTA_REG(16);
#undef PCS_DELTA_REG
  } else {
    int VS = p->vdim < 128 ? p->vdim : 128;
    while (VS > 8 && static_cast<size_t>(p->dim) * VS * sizeof(float) > 160 * 1024) VS /= 2;
    int R = 512 / VS;
    if (R < 1) R = 1;
    if (R > p->dim) R = p->dim;
    const int threads = ((VS * R + 31) / 32) * 32;
    const size_t smem = (static_cast<size_t>(p->dim) * VS + 3 * p->dim + VS + static_cast<size_t>(R) * VS) * sizeof(float);
    PCS_REQUIRE(smem <= 220 * 1024, "pcs_delta_scan: a state of %d rows exceeds shared memory", p->dim);
    if (smem > 48 * 1024)
      PCS_DISPATCH(p->dtype, PCS_CHECK_CUDA(cudaFuncSetAttribute(pcs::delta_scan_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024)));
    dim3 grid(p->n_seqs, p->heads, (p->vdim + VS - 1) / VS);
    PCS_DISPATCH(p->dtype, pcs::delta_scan_kernel<T><<<grid, threads, smem, st>>>(*p, VS, R));
  }
  PCS_CHECK_CUDA(cudaGetLastError());
  pcs::count_launch();
  return PCS_OK;
}

PCS_API int pcs_delta_chunk_prep(const pcs_delta_chunk_params* p, void* stream) {
  PCS_REQUIRE(p, "pcs_delta_chunk_prep: null params");
  if (p->n_chunks == 0) return PCS_OK;
  PCS_REQUIRE(p->ld || (p->dec_a && p->dt_bias && p->rate), "pcs_delta_chunk_prep: neither log decays per channel nor what per-head decays are formed of");
  PCS_REQUIRE(p->qk && p->v && p->b && p->chunk_first && p->chunk_len && p->qd && p->kd && p->w && p->g && p->u && p->a, "pcs_delta_chunk_prep: null tensor");
  PCS_REQUIRE(p->heads > 0 && p->heads <= 65535 && p->kv_heads > 0 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->dim <= 256 && p->vdim > 0,
              "pcs_delta_chunk_prep: bad sizes (dim %d of at most 256)", p->dim);
  const int D4 = (p->dim + 3) & ~3;
  const size_t smem = (static_cast<size_t>(2) * pcs::kC * (D4 + 4) + static_cast<size_t>(pcs::kC) * (D4 + 4 > pcs::kTi ? D4 + 4 : pcs::kTi) + 4 * D4 + pcs::kC * pcs::kC + pcs::kC) * sizeof(float);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (!p->ld) {
    const size_t smem_h = (static_cast<size_t>(2) * pcs::kC * (((p->dim + 31) & ~31) + 4) + pcs::kC * pcs::kC + 4 * pcs::kC + pcs::kC * pcs::kTi) * sizeof(float);
    PCS_DISPATCH(p->dtype, PCS_CHECK_CUDA(cudaFuncSetAttribute(pcs::delta_chunk_prep_head_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024)));
    PCS_DISPATCH(p->dtype, pcs::delta_chunk_prep_head_kernel<T><<<dim3(p->n_chunks, p->heads), pcs::kDpThreads, smem_h, st>>>(*p));
    PCS_CHECK_CUDA(cudaGetLastError());
    pcs::count_launch();
    return PCS_OK;
  }
  PCS_DISPATCH(p->dtype, PCS_CHECK_CUDA(cudaFuncSetAttribute(pcs::delta_chunk_prep_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024)));
  PCS_DISPATCH(p->dtype, pcs::delta_chunk_prep_kernel<T><<<dim3(p->n_chunks, p->heads), pcs::kDpThreads, smem, st>>>(*p));
  PCS_CHECK_CUDA(cudaGetLastError());
  pcs::count_launch();
  return PCS_OK;
}

PCS_API int pcs_delta_chunk_scan(const pcs_delta_chunk_params* p, void* stream) {
  PCS_REQUIRE(p, "pcs_delta_chunk_scan: null params");
  if (p->n_seqs == 0 || p->n_chunks == 0) return PCS_OK;
  PCS_REQUIRE(p->kd && p->w && p->g && p->u && p->s && p->s_pool && p->seq_slot && p->seq_pos0 && p->seq_chunk0 && p->seq_chunks, "pcs_delta_chunk_scan: null tensor");
  PCS_REQUIRE(p->heads > 0 && p->heads <= 65535 && p->n_seqs <= 65535 && p->dim > 0 && p->dim <= 256 && p->vdim > 0, "pcs_delta_chunk_scan: bad sizes");
  PCS_REQUIRE(((reinterpret_cast<uintptr_t>(p->kd) | reinterpret_cast<uintptr_t>(p->w)) & 15) == 0, "pcs_delta_chunk_scan: kd and w must be 16-byte aligned");
  const int L = (p->dim + 63) & ~63;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (p->dtype == PCS_BF16) return p->dim <= 128 ? pcs::launch_delta_chunk_scan_tc<1>(*p, st) : pcs::launch_delta_chunk_scan_tc<2>(*p, st);
  auto smem = [&](int vs, int nb) {
    return (static_cast<size_t>(nb) * (p->dim * pcs::kC + pcs::kC * L) + static_cast<size_t>(vs) * (L + pcs::kC + 8 * pcs::kC)) * sizeof(float);
  };
  // 8 columns per block where that still is one block per SM, else 16 (half of the chunk traffic); two buffers where they fit
  const long long rows = static_cast<long long>(p->heads) * p->n_seqs;
  const bool narrow = rows * ((p->vdim + 7) / 8) <= 148;
  const int vs = narrow ? 8 : 16;
  const bool one_wave = rows * ((p->vdim + vs - 1) / vs) <= 148;
  const bool two = smem(vs, 2) <= (one_wave ? 227u : 112u) * 1024u;
  if (narrow) return two ? pcs::launch_delta_chunk_scan<8, 2>(*p, smem(8, 2), st) : pcs::launch_delta_chunk_scan<8, 1>(*p, smem(8, 1), st);
  return two ? pcs::launch_delta_chunk_scan<16, 2>(*p, smem(16, 2), st) : pcs::launch_delta_chunk_scan<16, 1>(*p, smem(16, 1), st);
}

PCS_API int pcs_delta_chunk_out(const pcs_delta_chunk_params* p, const pcs_headnorm_params* o, void* stream) {
  PCS_REQUIRE(p && o, "pcs_delta_chunk_out: null params");
  if (p->n_chunks == 0) return PCS_OK;
  PCS_REQUIRE(p->qd && p->a && p->s && p->u && p->chunk_first && p->chunk_len && o->w && o->g && o->out, "pcs_delta_chunk_out: null tensor");
  PCS_REQUIRE(p->dtype == PCS_BF16 && p->heads > 0 && p->heads <= 65535 && p->dim > 0 && p->dim <= 256 && p->vdim > 0 && p->vdim <= 32 * pcs::kDoMaxWarps,
              "pcs_delta_chunk_out: serves bfloat16, dim up to 256 and vdim up to %d", 32 * pcs::kDoMaxWarps);
  PCS_REQUIRE(((reinterpret_cast<uintptr_t>(p->qd) | reinterpret_cast<uintptr_t>(p->a)) & 15) == 0, "pcs_delta_chunk_out: qd and a must be 16-byte aligned");
  const int warps = (p->vdim + 31) / 32 < 2 ? 2 : (p->vdim + 31) / 32, D16 = (p->dim + 15) & ~15;
  const size_t smem = static_cast<size_t>(2) * pcs::kC * (D16 + pcs::kC + 8) * sizeof(__nv_bfloat16) + static_cast<size_t>(warps) * pcs::kC * sizeof(float);
  PCS_CHECK_CUDA(cudaFuncSetAttribute(pcs::delta_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
  pcs::delta_chunk_out_kernel<<<dim3(p->n_chunks, p->heads), warps * 32, smem, static_cast<cudaStream_t>(stream)>>>(*p, *o);
  PCS_CHECK_CUDA(cudaGetLastError());
  pcs::count_launch();
  return PCS_OK;
}

PCS_API int pcs_head_norm_gate(const pcs_headnorm_params* p, void* stream) {
  PCS_REQUIRE(p, "pcs_head_norm_gate: null params");
  if (p->n_tokens == 0) return PCS_OK;
  PCS_REQUIRE(p->o && p->w && p->g && p->out && p->heads > 0 && p->vdim > 0 && (p->tok_row == nullptr || p->chunk_size > 0), "pcs_head_norm_gate: bad arguments");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const long long rows = static_cast<long long>(p->n_tokens) * p->heads;
  const int warps = rows < 8 * 148 ? 1 : 8;   // few rows: one warp per block
  PCS_DISPATCH(p->dtype, pcs::head_norm_gate_kernel<T><<<static_cast<unsigned>((rows + warps - 1) / warps), 32 * warps, 0, st>>>(*p));
  PCS_CHECK_CUDA(cudaGetLastError());
  pcs::count_launch();
  return PCS_OK;
}

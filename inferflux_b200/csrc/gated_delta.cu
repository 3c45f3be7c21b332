// The gated delta rule: a linear-attention state that shrinks by one factor per token and in which a key's old value is
// replaced by a new one, everything float32.  Per head, with S [dim x vdim] (zero at the start of a sequence), unit key k
// and unit, scaled query q (head h reads those of head h / (heads / kv_heads)):
//
//   g_t    = exp(-exp(A_log) * softplus(a_t + dt_bias))     beta_t = sigmoid(b_t)        a, b raw projections
//   S_t    = g_t S_{t-1} + k_t u_t^T,   u_t = beta_t (v_t - g_t S_{t-1}^T k_t)
//   o_t    = S_t^T q_t
//
// Portions.  Let c_i be the running sum of ln g from a segment's start, S the state there.  Unrolled over the segment,
//
//   S_i = e^(c_i) S + sum_{j <= i} e^(c_i - c_j) k_j u_j^T
//   (I + L) u = diag(beta) v - diag(beta e^c) K S,     L_ij = beta_i e^(c_i - c_j) (k_i . k_j)  for j < i
//
// so with W = (I + L)^-1 diag(beta e^c) K and U = (I + L)^-1 diag(beta) V, which do not depend on the state, u = U - W S.
// Three kernels:
//   1. a block a (segment, head): the running sums, L, and both triangular solves, a thread a column     (segments)
//   2. a block a (head, entry, 16 value columns): the segments one after the other: writes S, u = U - W S,
//      S <- e^(c_n) S + sum_j e^(c_n - c_j) k_j u_j^T; the last S goes into the slot                      (carry)
//   3. a block a (segment, head, 64 value columns): o_i = e^(c_i) S^T q_i + sum_{j <= i} e^(c_i - c_j) (q_i . k_j) u_j
// The sums c are of numbers below zero, and only differences c_i - c_j with j <= i are raised to e, so nothing overflows.
//
// A step of single tokens runs one kernel: a block a (head, entry, 32 value columns), eight threads a column, the
// column's state in registers between its read from the slot and its write.
#include "common.cuh"

#define IFX_GATED_DELTA_SEGMENT 32

namespace {
constexpr int SEG = IFX_GATED_DELTA_SEGMENT;
constexpr int VC = 16;                 // value columns of a carry block
constexpr int VT = 64;                 // value columns of an output block
constexpr int THREADS = 256;
constexpr int LLD = SEG + 4;           // row length of L and of the decayed scores in shared memory

struct GdArgs {
  const float* qkv; long long stride; int q_col, k_col, v_col;         // unit q (scaled) and k heads, v heads
  const float* raw; long long raw_stride; int a_col, b_col;            // the two raw projections, [row][heads] each
  const float* a_log; const float* dt_bias;                            // [heads]
  float* state;                                                        // [slots][heads][dim][vdim]
  const int* entry_q_start; const int* entry_q_len; const int* entry_slot;
  const int* seg_entry; const int* seg_t0; const int* entry_first_seg;
  int heads, kv_heads, dim, vdim, vec;                                 // vec: every staged row starts 16-byte aligned
  float* w_rows;                                                       // [row][heads * dim]
  float* u_rows;                                                       // [row][heads * vdim]
  float* cum;                                                          // [row][heads]
  float* seg_start;                                                    // [segments][heads][dim][vdim]
  float* out;                                                          // [row][heads * vdim]
};

__device__ __forceinline__ float log_decay(const GdArgs& p, int row, int h) {
  const float x = p.raw[(size_t)row * p.raw_stride + p.a_col + h] + p.dt_bias[h];
  return -expf(p.a_log[h]) * (fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))));
}
__device__ __forceinline__ float write_rate(const GdArgs& p, int row, int h) {
  return 1.0f / (1.0f + expf(-p.raw[(size_t)row * p.raw_stride + p.b_col + h]));
}

// Rows of keys and queries in shared memory: the head's size rounded up to a multiple of 4 (zeros behind it), four apart
// so that neighbouring rows fall into different banks.
__host__ __device__ __forceinline__ int padded(int dim) { return (dim + 3) & ~3; }
__host__ __device__ __forceinline__ int row_ld(int dim) { return padded(dim) + 4; }

// SEG rows of `width` floats from src (rows `stride` apart) into shared memory rows of `ld`, `fill` floats of each row
// written: zeros behind the width and behind row n.
__device__ __forceinline__ void stage_rows(float* dst, int ld, int fill, const float* src, long long stride, int n, int width,
                                           int vec, int tid) {
  if (vec) {
    const int per = fill >> 2;
    for (int idx = tid; idx < SEG * per; idx += THREADS) {
      const int j = idx / per, d = 4 * (idx - j * per);
      if (j < n && d < width) cp_async_f32x4(dst + j * ld + d, src + (size_t)j * stride + d);
      else *reinterpret_cast<float4*>(dst + j * ld + d) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
  } else {
    for (int idx = tid; idx < SEG * fill; idx += THREADS) {
      const int j = idx / fill, d = idx - j * fill;
      if (j < n && d < width) cp_async_f32(dst + j * ld + d, src + (size_t)j * stride + d);
      else dst[j * ld + d] = 0.0f;
    }
  }
}

// The thread's four dot products of rows bi, bi + 16 of a (16-byte aligned rows a_ld apart) with rows bj, bj + 16 of b.
__device__ __forceinline__ void dots_2x2(const float* a, int a_ld, const float* b, int b_ld, int dp, int bi, int bj, float (&d)[2][2]) {
  d[0][0] = d[0][1] = d[1][0] = d[1][1] = 0.0f;
  for (int n = 0; n < dp; n += 4) {
    const float4 a0 = *reinterpret_cast<const float4*>(a + bi * a_ld + n), a1 = *reinterpret_cast<const float4*>(a + (bi + 16) * a_ld + n);
    const float4 b0 = *reinterpret_cast<const float4*>(b + bj * b_ld + n), b1 = *reinterpret_cast<const float4*>(b + (bj + 16) * b_ld + n);
    d[0][0] = fmaf(a0.x, b0.x, fmaf(a0.y, b0.y, fmaf(a0.z, b0.z, fmaf(a0.w, b0.w, d[0][0]))));
    d[0][1] = fmaf(a0.x, b1.x, fmaf(a0.y, b1.y, fmaf(a0.z, b1.z, fmaf(a0.w, b1.w, d[0][1]))));
    d[1][0] = fmaf(a1.x, b0.x, fmaf(a1.y, b0.y, fmaf(a1.z, b0.z, fmaf(a1.w, b0.w, d[1][0]))));
    d[1][1] = fmaf(a1.x, b1.x, fmaf(a1.y, b1.y, fmaf(a1.z, b1.z, fmaf(a1.w, b1.w, d[1][1]))));
  }
}

__global__ void __launch_bounds__(THREADS)
gated_delta_segments_kernel(GdArgs p) {
  extern __shared__ __align__(16) float sm[];
  pdl_enter();
  const int D = p.dim, V = p.vdim, DP = padded(D), LD = row_ld(D);
  float* ks = sm;                          // [SEG][LD]
  float* L = ks + SEG * LD;                // [SEG][LLD]
  float* cs = L + SEG * LLD;               // [SEG] running sums of ln g
  float* be = cs + SEG;                    // [SEG] beta
  float* bg = be + SEG;                    // [SEG] beta e^c
  const int seg = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int e = p.seg_entry[seg], t0 = p.seg_t0[seg];
  const int n = min(SEG, p.entry_q_len[e] - t0), row0 = p.entry_q_start[e] + t0;
  const int kvh = h / (p.heads / p.kv_heads);
  stage_rows(ks, LD, DP, p.qkv + (size_t)row0 * p.stride + p.k_col + kvh * D, p.stride, n, D, p.vec, tid);
  cp_async_commit();
  if (tid < SEG) {                         // one warp: the running sums
    float c = tid < n ? log_decay(p, row0 + tid, h) : 0.0f;
    const float b = tid < n ? write_rate(p, row0 + tid, h) : 0.0f;
    for (int o = 1; o < SEG; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, c, o);
      if (tid >= o) c += up;
    }
    cs[tid] = c;
    be[tid] = b;
    bg[tid] = b * expf(c);
    if (tid < n) p.cum[(size_t)(row0 + tid) * p.heads + h] = c;
  }
  cp_async_wait_all();
  __syncthreads();
  {
    const int bi = tid >> 4, bj = tid & 15;
    float d[2][2];
    dots_2x2(ks, LD, ks, LD, DP, bi, bj, d);
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        const int i = bi + 16 * a, j = bj + 16 * b;
        L[i * LLD + j] = j < i ? be[i] * expf(cs[i] - cs[j]) * d[a][b] : 0.0f;
      }
  }
  __syncthreads();
  // both solves, a thread a column: x_i = rhs_i - sum_{j < i} L_ij x_j
  for (int c = tid; c < D + V; c += THREADS) {
    float x[SEG];
    if (c < D) {
#pragma unroll
      for (int i = 0; i < SEG; ++i) x[i] = bg[i] * ks[i * LD + c];
    } else {
      const float* v = p.qkv + (size_t)row0 * p.stride + p.v_col + h * V + (c - D);
#pragma unroll
      for (int i = 0; i < SEG; ++i) x[i] = i < n ? v[(size_t)i * p.stride] : 0.0f;
#pragma unroll
      for (int i = 0; i < SEG; ++i) x[i] *= be[i];
    }
    float* dst = c < D ? p.w_rows + (size_t)row0 * p.heads * D + h * D + c : p.u_rows + (size_t)row0 * p.heads * V + h * V + (c - D);
    const size_t step = (size_t)p.heads * (c < D ? D : V);
#pragma unroll
    for (int i = 0; i < SEG; ++i) {
      float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
      for (int j = 0; j < i; j += 4) {     // L is zero from the diagonal on, so a group of four may reach past it
        const float4 l = *reinterpret_cast<const float4*>(L + i * LLD + j);
        s0 = fmaf(l.x, x[j], s0);
        if (j + 1 < i) s1 = fmaf(l.y, x[j + 1], s1);
        if (j + 2 < i) s0 = fmaf(l.z, x[j + 2], s0);
        if (j + 3 < i) s1 = fmaf(l.w, x[j + 3], s1);
      }
      x[i] -= s0 + s1;
    }
#pragma unroll
    for (int i = 0; i < SEG; ++i)
      if (i < n) dst[(size_t)i * step] = x[i];
  }
}

__global__ void __launch_bounds__(THREADS)
gated_delta_carry_kernel(GdArgs p) {
  extern __shared__ __align__(16) float sm[];
  pdl_enter();
  const int D = p.dim, V = p.vdim, DP = padded(D), LD = row_ld(D);
  const int BUF = 2 * SEG * LD + SEG * VC + SEG;
  float* St = sm;                          // [VC][LD]: the state's columns, key rows side by side
  float* us = St + VC * LD;                // [SEG][VC]: u, each times what is left of it at the segment's end
  float* bufs = us + SEG * VC;             // two of: W [SEG][LD], K [SEG][LD], U [SEG][VC], c [SEG]
  const int h = blockIdx.x, e = blockIdx.y, v0 = blockIdx.z * VC, tid = threadIdx.x;
  const int len = p.entry_q_len[e], r0 = p.entry_q_start[e];
  const int n_seg = (len + SEG - 1) / SEG, seg0 = p.entry_first_seg[e];
  const int kvh = h / (p.heads / p.kv_heads);
  const int vcols = min(VC, V - v0);
  float* slot = p.state + ((size_t)p.entry_slot[e] * p.heads + h) * D * V;
  auto stage = [&](int s, float* buf) {
    const int row = r0 + s * SEG, n = min(SEG, len - s * SEG);
    stage_rows(buf, LD, DP, p.w_rows + ((size_t)row * p.heads + h) * D, (long long)p.heads * D, n, D, p.vec, tid);
    stage_rows(buf + SEG * LD, LD, DP, p.qkv + (size_t)row * p.stride + p.k_col + kvh * D, p.stride, n, D, p.vec, tid);
    stage_rows(buf + 2 * SEG * LD, VC, VC, p.u_rows + ((size_t)row * p.heads + h) * V + v0, (long long)p.heads * V, n, vcols,
               p.vec && !(vcols & 3), tid);
    if (tid < SEG) {
      float* c = buf + 2 * SEG * LD + SEG * VC + tid;
      if (tid < n) cp_async_f32(c, p.cum + (size_t)(row + tid) * p.heads + h);
      else *c = 0.0f;
    }
    cp_async_commit();
  };
  if (n_seg > 0) stage(0, bufs);
  for (int idx = tid; idx < DP * VC; idx += THREADS) {
    const int d = idx / VC, c = idx - d * VC;
    St[c * LD + d] = (d < D && c < vcols) ? slot[(size_t)d * V + v0 + c] : 0.0f;
  }
  for (int s = 0; s < n_seg; ++s) {
    float* W = bufs + (s & 1) * BUF;
    const float* K = W + SEG * LD;
    const float* U = K + SEG * LD;
    const float* cs = U + SEG * VC;
    const int n = min(SEG, len - s * SEG), row = r0 + s * SEG;
    cp_async_wait_all();
    __syncthreads();                       // this segment's rows are here and the state is whole
    if (s + 1 < n_seg) stage(s + 1, bufs + ((s + 1) & 1) * BUF);
    float* start = p.seg_start + ((size_t)(seg0 + s) * p.heads + h) * D * V + v0;
    for (int idx = tid; idx < D * VC; idx += THREADS) {
      const int d = idx / VC, c = idx - d * VC;
      if (c < vcols) start[(size_t)d * V + c] = St[c * LD + d];
    }
    {                                      // u = U - W S: rows ip and ip + 16, one column
      const int c = tid & 15, ip = tid >> 4;
      float a0 = 0.0f, a1 = 0.0f, b0 = 0.0f, b1 = 0.0f;
#pragma unroll 4
      for (int d = 0; d < DP; d += 4) {
        const float4 x = *reinterpret_cast<const float4*>(St + c * LD + d);
        const float4 w0 = *reinterpret_cast<const float4*>(W + ip * LD + d), w1 = *reinterpret_cast<const float4*>(W + (ip + 16) * LD + d);
        a0 = fmaf(w0.x, x.x, fmaf(w0.y, x.y, a0));
        a1 = fmaf(w0.z, x.z, fmaf(w0.w, x.w, a1));
        b0 = fmaf(w1.x, x.x, fmaf(w1.y, x.y, b0));
        b1 = fmaf(w1.z, x.z, fmaf(w1.w, x.w, b1));
      }
      const float ua = U[ip * VC + c] - (a0 + a1), ub = U[(ip + 16) * VC + c] - (b0 + b1);
      const float last = cs[n - 1];
      us[ip * VC + c] = ip < n ? ua * expf(last - cs[ip]) : 0.0f;
      us[(ip + 16) * VC + c] = ip + 16 < n ? ub * expf(last - cs[ip + 16]) : 0.0f;
      if (c < vcols) {
        float* dst = p.u_rows + ((size_t)row * p.heads + h) * V + v0 + c;
        if (ip < n) dst[(size_t)ip * p.heads * V] = ua;
        if (ip + 16 < n) dst[(size_t)(ip + 16) * p.heads * V] = ub;
      }
    }
    __syncthreads();
    {                                      // S <- e^(c_n) S + sum_j k_j us_j: two columns, four key rows
      const int c = 2 * (tid & 7);
      const float g = expf(cs[n - 1]);
      for (int d = 4 * (tid >> 3); d < DP; d += 4 * (THREADS / 8)) {
        float4 sa = *reinterpret_cast<float4*>(St + c * LD + d), sb = *reinterpret_cast<float4*>(St + (c + 1) * LD + d);
        sa.x *= g; sa.y *= g; sa.z *= g; sa.w *= g;
        sb.x *= g; sb.y *= g; sb.z *= g; sb.w *= g;
#pragma unroll 4
        for (int j = 0; j < n; ++j) {
          const float4 k = *reinterpret_cast<const float4*>(K + j * LD + d);
          const float2 u = *reinterpret_cast<const float2*>(us + j * VC + c);
          sa.x = fmaf(k.x, u.x, sa.x); sa.y = fmaf(k.y, u.x, sa.y); sa.z = fmaf(k.z, u.x, sa.z); sa.w = fmaf(k.w, u.x, sa.w);
          sb.x = fmaf(k.x, u.y, sb.x); sb.y = fmaf(k.y, u.y, sb.y); sb.z = fmaf(k.z, u.y, sb.z); sb.w = fmaf(k.w, u.y, sb.w);
        }
        *reinterpret_cast<float4*>(St + c * LD + d) = sa;
        *reinterpret_cast<float4*>(St + (c + 1) * LD + d) = sb;
      }
    }
  }
  __syncthreads();
  for (int idx = tid; idx < D * VC; idx += THREADS) {
    const int d = idx / VC, c = idx - d * VC;
    if (c < vcols) slot[(size_t)d * V + v0 + c] = St[c * LD + d];
  }
}

__global__ void __launch_bounds__(THREADS)
gated_delta_outputs_kernel(GdArgs p) {
  extern __shared__ __align__(16) float sm[];
  pdl_enter();
  const int D = p.dim, V = p.vdim, DP = padded(D), LD = row_ld(D);
  float* ks = sm;                          // [SEG][LD]
  float* qs = ks + SEG * LD;               // [SEG][LD]
  float* us = qs + SEG * LD;               // [SEG][VT]
  float* St = us + SEG * VT;               // [DP][VT]
  float* P = St + DP * VT;                 // [SEG][LLD]
  float* cs = P + SEG * LLD;               // [SEG]
  const int seg = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT, tid = threadIdx.x;
  const int e = p.seg_entry[seg], t0 = p.seg_t0[seg];
  const int n = min(SEG, p.entry_q_len[e] - t0), row0 = p.entry_q_start[e] + t0;
  const int kvh = h / (p.heads / p.kv_heads), vcols = min(VT, V - v0);
  const float* rows = p.qkv + (size_t)row0 * p.stride + kvh * D;
  stage_rows(ks, LD, DP, rows + p.k_col, p.stride, n, D, p.vec, tid);
  stage_rows(qs, LD, DP, rows + p.q_col, p.stride, n, D, p.vec, tid);
  stage_rows(us, VT, VT, p.u_rows + ((size_t)row0 * p.heads + h) * V + v0, (long long)p.heads * V, n, vcols, p.vec && !(vcols & 3), tid);
  const float* start = p.seg_start + ((size_t)seg * p.heads + h) * D * V + v0;
  if (p.vec && !(vcols & 3)) {
    for (int idx = tid; idx < DP * (VT / 4); idx += THREADS) {
      const int d = idx / (VT / 4), c = 4 * (idx - d * (VT / 4));
      if (c < vcols) cp_async_f32x4(St + d * VT + c, start + (size_t)d * V + c);
      else *reinterpret_cast<float4*>(St + d * VT + c) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
  } else {
    for (int idx = tid; idx < DP * VT; idx += THREADS) {
      const int d = idx / VT, c = idx - d * VT;
      St[idx] = (d < D && c < vcols) ? start[(size_t)d * V + c] : 0.0f;
    }
  }
  cp_async_commit();
  if (tid < SEG) cs[tid] = tid < n ? p.cum[(size_t)(row0 + tid) * p.heads + h] : 0.0f;
  cp_async_wait_all();
  __syncthreads();
  {                                        // P_ij = e^(c_i - c_j) (q_i . k_j) for j <= i
    const int bi = tid >> 4, bj = tid & 15;
    float d[2][2];
    dots_2x2(qs, LD, ks, LD, DP, bi, bj, d);
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        const int i = bi + 16 * a, j = bj + 16 * b;
        P[i * LLD + j] = (j <= i && i < n) ? d[a][b] * expf(cs[i] - cs[j]) : 0.0f;
      }
  }
  __syncthreads();
  // a thread owns tokens tg, tg + 16 and four columns
  const int cg = 4 * (tid & 15), tg = tid >> 4;
  float inter[2][4] = {}, intra[2][4] = {};
  for (int d = 0; d < DP; d += 4) {
    const float4 qa = *reinterpret_cast<const float4*>(qs + tg * LD + d), qb = *reinterpret_cast<const float4*>(qs + (tg + 16) * LD + d);
    const float qv[2][4] = {{qa.x, qa.y, qa.z, qa.w}, {qb.x, qb.y, qb.z, qb.w}};
#pragma unroll
    for (int r = 0; r < 4; ++r) {
      const float4 s4 = *reinterpret_cast<const float4*>(St + (d + r) * VT + cg);
      const float sv[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
      for (int a = 0; a < 2; ++a)
#pragma unroll
        for (int b = 0; b < 4; ++b) inter[a][b] = fmaf(qv[a][r], sv[b], inter[a][b]);
    }
  }
  for (int j = 0; j < n; ++j) {
    const float4 u4 = *reinterpret_cast<const float4*>(us + j * VT + cg);
    const float uv[4] = {u4.x, u4.y, u4.z, u4.w};
    const float pa = P[tg * LLD + j], pb = P[(tg + 16) * LLD + j];
#pragma unroll
    for (int b = 0; b < 4; ++b) { intra[0][b] = fmaf(pa, uv[b], intra[0][b]); intra[1][b] = fmaf(pb, uv[b], intra[1][b]); }
  }
#pragma unroll
  for (int a = 0; a < 2; ++a) {
    const int i = tg + 16 * a;
    if (i >= n) continue;
    const float g = expf(cs[i]);
    float* dst = p.out + ((size_t)(row0 + i) * p.heads + h) * V + v0 + cg;
#pragma unroll
    for (int b = 0; b < 4; ++b)
      if (cg + b < vcols) dst[b] = fmaf(g, inter[a][b], intra[a][b]);
  }
}

// Single tokens: NI key rows a thread, g + 8 i of the block's head.
template <int NI>
__global__ void __launch_bounds__(256)
gated_delta_step_kernel(GdArgs p) {
  __shared__ float ks[8 * NI], qs[8 * NI], red[8][33];
  pdl_enter();
  const int h = blockIdx.x, e = blockIdx.y, tid = threadIdx.x, lane = tid & 31, grp = tid >> 5;
  const int c = blockIdx.z * 32 + lane, D = p.dim, V = p.vdim;
  const int row = p.entry_q_start[e], kvh = h / (p.heads / p.kv_heads);
  const bool on = c < V;
  float* st = p.state + ((size_t)p.entry_slot[e] * p.heads + h) * D * V + (on ? c : 0);
  float S[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = grp + 8 * i;
    S[i] = (on && d < D) ? st[(size_t)d * V] : 0.0f;
  }
  const float* r = p.qkv + (size_t)row * p.stride;
  for (int d = tid; d < 8 * NI; d += 256) {
    ks[d] = d < D ? r[p.k_col + kvh * D + d] : 0.0f;
    qs[d] = d < D ? r[p.q_col + kvh * D + d] : 0.0f;
  }
  const float v = on ? r[p.v_col + h * V + c] : 0.0f;
  const float g = expf(log_decay(p, row, h)), beta = write_rate(p, row, h);
  __syncthreads();
  float dot = 0.0f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    S[i] *= g;
    dot = fmaf(ks[grp + 8 * i], S[i], dot);
  }
  red[grp][lane] = dot;
  __syncthreads();
  dot = 0.0f;
#pragma unroll
  for (int w = 0; w < 8; ++w) dot += red[w][lane];
  const float u = beta * (v - dot);
  float o = 0.0f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = grp + 8 * i;
    S[i] = fmaf(ks[d], u, S[i]);
    o = fmaf(qs[d], S[i], o);
    if (on && d < D) st[(size_t)d * V] = S[i];
  }
  __syncthreads();
  red[grp][lane] = o;
  __syncthreads();
  if (grp == 0 && on) {
    o = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) o += red[w][lane];
    p.out[((size_t)row * p.heads + h) * V + c] = o;
  }
}

size_t segments_smem(int D) { return ((size_t)SEG * row_ld(D) + SEG * LLD + 3 * SEG) * sizeof(float); }
size_t carry_smem(int D) { return ((size_t)VC * row_ld(D) + SEG * VC + 2 * (2 * (size_t)SEG * row_ld(D) + SEG * VC + SEG)) * sizeof(float); }
size_t outputs_smem(int D) {
  return (2 * (size_t)SEG * row_ld(D) + SEG * VT + (size_t)padded(D) * VT + SEG * LLD + SEG) * sizeof(float);
}
constexpr int MAX_DIM = 256;
}  // namespace

IFX_API int ifx_gated_delta_segment() { return SEG; }

// qkv float32 rows: unit, scaled q heads and unit k heads (kv_heads * dim each), v heads (heads * vdim) from the given
// columns on; raw float32 rows: the decay's and the rate's projections from a_col and b_col on, [heads] each;
// state float32 [slots][heads][dim][vdim]; out float32 [N][heads * vdim].  n_segments 0: every entry brings one token.
// Otherwise w_rows [N][heads * dim], u_rows [N][heads * vdim], cum [N][heads] and seg_start [segments][heads][dim][vdim]
// (float32) are scratch, and the segments of IFX_GATED_DELTA_SEGMENT tokens are listed entry by entry.
IFX_API int ifx_gated_delta_scan(const float* qkv, long long stride, int q_col, int k_col, int v_col, const float* raw,
                                 long long raw_stride, int a_col, int b_col, const float* a_log, const float* dt_bias,
                                 float* state, const int* entry_q_start, const int* entry_q_len, const int* entry_slot,
                                 int n_entries, const int* seg_entry, const int* seg_t0, const int* entry_first_seg,
                                 int n_segments, float* w_rows, float* u_rows, float* cum, float* seg_start, float* out,
                                 int heads, int kv_heads, int dim, int vdim, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  if (heads < 1 || kv_heads < 1 || heads % kv_heads || dim < 1 || dim > MAX_DIM || vdim < 1 || heads > 65535 || n_entries > 65535)
    return IFX_ERR_UNSUPPORTED;
  GdArgs p{qkv, stride, q_col, k_col, v_col, raw, raw_stride, a_col, b_col, a_log, dt_bias, state, entry_q_start, entry_q_len,
           entry_slot, seg_entry, seg_t0, entry_first_seg, heads, kv_heads, dim, vdim, 0, w_rows, u_rows, cum, seg_start, out};
  p.vec = !((dim | vdim | q_col | k_col | v_col) & 3) && !(stride & 3) &&
          !(((uintptr_t)qkv | (uintptr_t)w_rows | (uintptr_t)u_rows | (uintptr_t)seg_start) & 15);
  int rc;
  if (n_segments <= 0) {
    const dim3 grid(heads, n_entries, (vdim + 31) / 32);
    if (dim <= 32) rc = launch_pdl(gated_delta_step_kernel<4>, grid, dim3(256), 0, stream, p);
    else if (dim <= 64) rc = launch_pdl(gated_delta_step_kernel<8>, grid, dim3(256), 0, stream, p);
    else if (dim <= 128) rc = launch_pdl(gated_delta_step_kernel<16>, grid, dim3(256), 0, stream, p);
    else rc = launch_pdl(gated_delta_step_kernel<32>, grid, dim3(256), 0, stream, p);
    return rc ? rc : IFX_LAUNCH_CHECK();
  }
  if (!w_rows || !u_rows || !cum || !seg_start) return IFX_ERR_UNSUPPORTED;
  static bool attr_done = false;
  if (!attr_done) {
    cudaError_t err = cudaFuncSetAttribute(gated_delta_carry_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)carry_smem(MAX_DIM));
    if (err == cudaSuccess)
      err = cudaFuncSetAttribute(gated_delta_outputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)outputs_smem(MAX_DIM));
    if (err == cudaSuccess)
      err = cudaFuncSetAttribute(gated_delta_segments_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)segments_smem(MAX_DIM));
    if (err != cudaSuccess) return (int)err;
    attr_done = true;
  }
  rc = launch_pdl(gated_delta_segments_kernel, dim3(n_segments, heads), dim3(THREADS), segments_smem(dim), stream, p);
  if (!rc) rc = launch_pdl(gated_delta_carry_kernel, dim3(heads, n_entries, (vdim + VC - 1) / VC), dim3(THREADS), carry_smem(dim), stream, p);
  if (!rc) rc = launch_pdl(gated_delta_outputs_kernel, dim3(n_segments, heads, (vdim + VT - 1) / VT), dim3(THREADS), outputs_smem(dim), stream, p);
  return rc ? rc : IFX_LAUNCH_CHECK();
}

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
//   1. a block a (segment, head): the running sums, L, and both triangular solves, a thread a column
//   2. the segments one after the other: each one's starting S, u = U - W S, and the S that the next one starts from
//   3. every segment's outputs from its starting S                    (2 and 3: segment_scan.cuh)
// The sums c are of numbers below zero, and only differences c_i - c_j with j <= i are raised to e, so nothing overflows.
//
// One decay per head and key channel (dec given: g_t is then a diagonal, g_t[d] = exp(-exp(A_log) softplus(dec_t[h][d] +
// dt_bias[h][d])), and c_i a vector): the same equations with the exponentials inside the dot products,
//
//   L_ij = beta_i sum_d k_i[d] e^(c_i[d] - c_j[d]) k_j[d],   W = (I + L)^-1 diag(beta) (e^(c) K)
//   S_n  = diag(e^(c_n)) S + sum_j (e^(c_n - c_j) k_j) u_j^T,   o_i = (e^(c_i) q_i)^T S + sum_j (q_i e^(c_i - c_j) k_j) u_j
//
// The differences are taken pair by pair and channel by channel, so decays of any strength stay finite here too.  The
// first kernel leaves behind what the other two multiply: e^(c_n - c_j) k_j, e^(c_i) q_i, e^(c_n) and the scores' table.
//
// A step of single tokens runs one kernel: a block a (head, entry, 32 value columns), eight threads a column, the
// column's state in registers between its read from the slot and its write.
#include "segment_scan.cuh"

namespace {
using segscan::SEG;
using segscan::row_ld;
constexpr int THREADS = 256;
constexpr int LLD = SEG + 4;           // row length of L in shared memory

struct GdArgs {
  const float* qkv; long long stride; int q_col, k_col, v_col;         // unit q (scaled) and k heads, v heads
  const float* raw; long long raw_stride; int a_col, b_col;            // the two raw projections, [row][heads] each
  const float* dec; long long dec_stride;                              // or: the decays' projection, [row][heads * dim]
  const float* a_log; const float* dt_bias;                            // [heads]; with dec: dt_bias [heads * dim]
  float* state;                                                        // [slots][heads][dim][vdim]
  const int* entry_q_start; const int* entry_q_len; const int* entry_slot;
  const int* seg_entry; const int* seg_t0; const int* entry_first_seg;
  int heads, kv_heads, dim, vdim, vec;                                 // vec: every staged row starts 16-byte aligned
  float* w_rows;                                                       // [row][heads * dim]
  float* u_rows;                                                       // [row][heads * vdim]
  float* cum;                                                          // [row][heads]
  float* k_rows; float* q_rows;                                        // with dec: [row][heads * dim] each
  float* seg_decay;                                                    // with dec: [segments][heads][dim]
  float* scores;                                                       // with dec: [segments][heads][SEG j][SEG i]
  float* out;                                                          // [row][heads * vdim]
};

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float log_decay(const GdArgs& p, int row, int h) {
  return -expf(p.a_log[h]) * softplus(p.raw[(size_t)row * p.raw_stride + p.a_col + h] + p.dt_bias[h]);
}
__device__ __forceinline__ float write_rate(const GdArgs& p, int row, int h) {
  return 1.0f / (1.0f + expf(-p.raw[(size_t)row * p.raw_stride + p.b_col + h]));
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

// x <- (I + L)^-1 x for a thread's column of SEG numbers; L zero from the diagonal on, rows LLD apart
__device__ __forceinline__ void solve_column(const float* L, float (&x)[SEG]) {
#pragma unroll
  for (int i = 0; i < SEG; ++i) {
    float s0 = 0.0f, s1 = 0.0f;
#pragma unroll
    for (int j = 0; j < i; j += 4) {       // a group of four may reach past the diagonal
      const float4 l = *reinterpret_cast<const float4*>(L + i * LLD + j);
      s0 = fmaf(l.x, x[j], s0);
      if (j + 1 < i) s1 = fmaf(l.y, x[j + 1], s1);
      if (j + 2 < i) s0 = fmaf(l.z, x[j + 2], s0);
      if (j + 3 < i) s1 = fmaf(l.w, x[j + 3], s1);
    }
    x[i] -= s0 + s1;
  }
}

__global__ void __launch_bounds__(THREADS)
gated_delta_segments_kernel(GdArgs p) {
  extern __shared__ __align__(16) float sm[];
  pdl_enter();
  const int D = p.dim, V = p.vdim, DP = segscan::pad4(D), LD = row_ld(D);
  float* ks = sm;                          // [SEG][LD]
  float* L = ks + SEG * LD;                // [SEG][LLD]
  float* cs = L + SEG * LLD;               // [SEG] running sums of ln g
  float* be = cs + SEG;                    // [SEG] beta
  float* bg = be + SEG;                    // [SEG] beta e^c
  const int seg = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int e = p.seg_entry[seg], t0 = p.seg_t0[seg];
  const int n = min(SEG, p.entry_q_len[e] - t0), row0 = p.entry_q_start[e] + t0;
  const int kvh = h / (p.heads / p.kv_heads);
  segscan::stage_rows(ks, LD, DP, p.qkv + (size_t)row0 * p.stride + p.k_col + kvh * D, p.stride, n, D, p.vec, tid, THREADS);
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
    solve_column(L, x);
#pragma unroll
    for (int i = 0; i < SEG; ++i)
      if (i < n) dst[(size_t)i * step] = x[i];
  }
}

// Single tokens: NI key rows a thread, g + 8 i of the block's head.
template <int NI, bool CHANNEL>
__global__ void __launch_bounds__(256)
gated_delta_step_kernel(GdArgs p) {
  __shared__ float ks[8 * NI], qs[8 * NI], gs[CHANNEL ? 8 * NI : 1], red[8][33];
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
    if (CHANNEL)
      gs[d] = d < D ? expf(-expf(p.a_log[h]) * softplus(p.dec[(size_t)row * p.dec_stride + h * D + d] + p.dt_bias[h * D + d])) : 0.0f;
  }
  const float v = on ? r[p.v_col + h * V + c] : 0.0f;
  const float g = CHANNEL ? 1.0f : expf(log_decay(p, row, h)), beta = write_rate(p, row, h);
  __syncthreads();
  float dot = 0.0f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    S[i] *= CHANNEL ? gs[grp + 8 * i] : g;
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

// One decay per key channel.  The logarithms' running sums c are kept to base two.  Between the segment's halves the
// exponentials factor: with m the sum at the first half's end, e^(c_i - c_j) = e^(c_i - m) e^(m - c_j) for i in the second and
// j in the first half, neither factor above one, so a quarter of the pairs' square is a product of scaled rows; inside the
// halves the differences are taken pair by pair.
__global__ void __launch_bounds__(THREADS, 2)
channel_delta_segments_kernel(GdArgs p) {
  extern __shared__ __align__(16) float sm[];
  pdl_enter();
  constexpr int HALF = SEG / 2, EACH = SEG / (THREADS / 32);
  const int D = p.dim, V = p.vdim, DP = segscan::pad4(D), LD = row_ld(D);
  float* ks = sm;                          // [SEG][LD]
  float* qs = ks + SEG * LD;               // [SEG][LD]
  float* cs = qs + SEG * LD;               // [SEG][LD] running sums of log2 g per channel
  float* km = cs + SEG * LD;               // [SEG][LD] keys: times e^(m - c) in the first half, e^(c - m) in the second
  float* qm = km + SEG * LD;               // [HALF][LD] the second half's queries times e^(c - m)
  float* L = qm + HALF * LD;               // [SEG][LLD]
  float* A = L + SEG * LLD;                // [SEG j][LLD] scores, transposed
  float* be = A + SEG * LLD;               // [SEG] beta
  const int seg = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int e = p.seg_entry[seg], t0 = p.seg_t0[seg];
  const int n = min(SEG, p.entry_q_len[e] - t0), row0 = p.entry_q_start[e] + t0;
  const int kvh = h / (p.heads / p.kv_heads);
  segscan::stage_rows(ks, LD, DP, p.qkv + (size_t)row0 * p.stride + p.k_col + kvh * D, p.stride, n, D, p.vec, tid, THREADS);
  segscan::stage_rows(qs, LD, DP, p.qkv + (size_t)row0 * p.stride + p.q_col + kvh * D, p.stride, n, D, p.vec, tid, THREADS);
  cp_async_commit();
  {
    const float rate = -1.4426950408889634f * expf(p.a_log[h]);
    const float* dec = p.dec + (size_t)row0 * p.dec_stride + h * D;
    const float* bias = p.dt_bias + h * D;
    const int i0 = tid >> 5;
    for (int d = tid & 31; d < DP; d += 32) {
      float x[EACH];
#pragma unroll
      for (int u = 0; u < EACH; ++u) {
        const int i = i0 + u * (THREADS / 32);
        x[u] = i < n && d < D ? dec[(size_t)i * p.dec_stride + d] : 0.0f;
      }
      const float bd = d < D ? bias[d] : 0.0f;
#pragma unroll
      for (int u = 0; u < EACH; ++u) {
        const int i = i0 + u * (THREADS / 32);
        cs[i * LD + d] = i < n && d < D ? rate * softplus(x[u] + bd) : 0.0f;
      }
    }
  }
  if (tid < SEG) be[tid] = tid < n ? write_rate(p, row0 + tid, h) : 0.0f;
  for (int idx = tid; idx < SEG * LLD; idx += THREADS) L[idx] = A[idx] = 0.0f;
  __syncthreads();
  for (int d = tid; d < DP; d += THREADS) {
    float x[SEG];
#pragma unroll
    for (int i = 0; i < SEG; ++i) x[i] = cs[i * LD + d];
#pragma unroll
    for (int i = 1; i < SEG; ++i) x[i] += x[i - 1];
#pragma unroll
    for (int i = 0; i < SEG; ++i) cs[i * LD + d] = x[i];
  }
  cp_async_wait_all();
  __syncthreads();
  auto at = [&](const float* b, int i, int d) { return *reinterpret_cast<const float4*>(b + i * LD + d); };
  auto put = [&](float* b, int i, int d, float4 v) { *reinterpret_cast<float4*>(b + i * LD + d) = v; };
  auto times = [](float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); };
  auto apart = [](float4 a, float4 b) { return make_float4(exp2f(a.x - b.x), exp2f(a.y - b.y), exp2f(a.z - b.z), exp2f(a.w - b.w)); };
  auto dot = [](float4 a, float4 b, float s) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, s)))); };
  // the scaled rows; eight neighbouring threads walk a row
  for (int i = tid >> 3; i < SEG; i += THREADS / 8)
    for (int d = 4 * (tid & 7); d < DP; d += 32) {
      const float4 c = at(cs, i, d), m = at(cs, HALF - 1, d);
      if (i < HALF) {
        put(km, i, d, times(at(ks, i, d), apart(m, c)));
      } else {
        const float4 g = apart(c, m);
        put(km, i, d, times(at(ks, i, d), g));
        put(qm, i - HALF, d, times(at(qs, i, d), g));
      }
    }
  {
    // inside the halves: the pair (bi, bj) of the first half where bj <= bi, else (bj, bi) of the second, a thread one pair;
    // the second half's diagonal (scores only, no decay in them) by sixteen threads a row
    const int bi = tid >> 4, bj = tid & 15;
    const bool first = bj <= bi;
    const int i = first ? bi : HALF + bj, j = first ? bj : HALF + bi;
    float kk = 0.0f, qk = 0.0f, own = 0.0f;
#pragma unroll 4
    for (int d = 0; d < DP; d += 4) {
      const float4 t = times(at(ks, j, d), apart(at(cs, i, d), at(cs, j, d)));
      kk = dot(at(ks, i, d), t, kk);
      qk = dot(at(qs, i, d), t, qk);
    }
    for (int d = 4 * bj; d < DP; d += 64) own = dot(at(ks, HALF + bi, d), at(qs, HALF + bi, d), own);
    for (int o = 8; o > 0; o >>= 1) own += __shfl_xor_sync(0xffffffffu, own, o);
    if (j < i) L[i * LLD + j] = be[i] * kk;
    A[j * LLD + i] = qk;
    if (bj == 0) A[(HALF + bi) * LLD + HALF + bi] = own;
  }
  __syncthreads();
  {
    // the second half's rows with the first half's
    const int bi = tid >> 4, bj = tid & 15, i = HALF + bi;
    float kk = 0.0f, qk = 0.0f;
#pragma unroll 4
    for (int d = 0; d < DP; d += 4) {
      const float4 kj = at(km, bj, d);
      kk = dot(at(km, i, d), kj, kk);
      qk = dot(at(qm, bi, d), kj, qk);
    }
    L[i * LLD + bj] = be[i] * kk;
    A[bj * LLD + i] = qk;
  }
  __syncthreads();                         // km has been read: its place takes the keys times e^c
  for (int i = tid >> 3; i < SEG; i += THREADS / 8)
    for (int d = 4 * (tid & 7); d < DP; d += 32) {
      const float4 c = at(cs, i, d), last = at(cs, n - 1, d), k = at(ks, i, d);
      const float4 g = apart(c, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
      put(km, i, d, times(k, g));
      if (i >= n) continue;
      const float4 kr = times(k, apart(last, c)), qr = times(at(qs, i, d), g);
      const size_t to = ((size_t)(row0 + i) * p.heads + h) * D + d;
      if (p.vec) {
        *reinterpret_cast<float4*>(p.k_rows + to) = kr;
        *reinterpret_cast<float4*>(p.q_rows + to) = qr;
      } else {
        const float kv[4] = {kr.x, kr.y, kr.z, kr.w}, qv[4] = {qr.x, qr.y, qr.z, qr.w};
#pragma unroll
        for (int x = 0; x < 4; ++x)
          if (d + x < D) { p.k_rows[to + x] = kv[x]; p.q_rows[to + x] = qv[x]; }
      }
    }
  for (int d = tid; d < D; d += THREADS) p.seg_decay[((size_t)seg * p.heads + h) * D + d] = exp2f(cs[(n - 1) * LD + d]);
  {
    float* dst = p.scores + ((size_t)seg * p.heads + h) * SEG * SEG;
    const int j = tid >> 3, i = 4 * (tid & 7);
    *reinterpret_cast<float4*>(dst + j * SEG + i) = *reinterpret_cast<const float4*>(A + j * LLD + i);
  }
  __syncthreads();
  for (int c = tid; c < D + V; c += THREADS) {
    float x[SEG];
    if (c < D) {
#pragma unroll
      for (int i = 0; i < SEG; ++i) x[i] = be[i] * km[i * LD + c];
    } else {
      const float* v = p.qkv + (size_t)row0 * p.stride + p.v_col + h * V + (c - D);
#pragma unroll
      for (int i = 0; i < SEG; ++i) x[i] = i < n ? v[(size_t)i * p.stride] : 0.0f;
#pragma unroll
      for (int i = 0; i < SEG; ++i) x[i] *= be[i];
    }
    float* dst = c < D ? p.w_rows + (size_t)row0 * p.heads * D + h * D + c : p.u_rows + (size_t)row0 * p.heads * V + h * V + (c - D);
    const size_t step = (size_t)p.heads * (c < D ? D : V);
    solve_column(L, x);
#pragma unroll
    for (int i = 0; i < SEG; ++i)
      if (i < n) dst[(size_t)i * step] = x[i];
  }
}

size_t channel_segments_smem(int D) { return ((size_t)(4 * SEG + SEG / 2) * row_ld(D) + 2 * SEG * LLD + SEG) * sizeof(float); }
size_t segments_smem(int D) { return ((size_t)SEG * row_ld(D) + SEG * LLD + 3 * SEG) * sizeof(float); }
}  // namespace

IFX_API int ifx_gated_delta_segment() { return SEG; }

// qkv float32 rows: unit, scaled q heads and unit k heads (kv_heads * dim each), v heads (heads * vdim) from the given
// columns on; raw float32 rows: the decay's and the rate's projections from a_col and b_col on, [heads] each;
// state float32 [slots][heads][dim][vdim]; out float32 [N][heads * vdim].  n_segments 0: every entry brings one token.
// Otherwise w_rows [N][heads * dim], u_rows [N][heads * vdim], cum [N][heads] and seg_start [segments][heads][dim][vdim]
// (float32) are scratch, and the segments of ifx_gated_delta_segment() tokens are listed entry by entry.
// dec (or null): float32 rows of heads * dim, the projection of one decay per head and key channel; raw's a_col is not
// read then, dt_bias is [heads * dim], and k_rows, q_rows [N][heads * dim], seg_decay [segments][heads][dim] and scores
// [segments][heads][32][32] are scratch in cum's place.
IFX_API int ifx_gated_delta_scan(const float* qkv, long long stride, int q_col, int k_col, int v_col, const float* raw,
                                 long long raw_stride, int a_col, int b_col, const float* dec, long long dec_stride,
                                 const float* a_log, const float* dt_bias,
                                 float* state, const int* entry_q_start, const int* entry_q_len, const int* entry_slot,
                                 int n_entries, const int* seg_entry, const int* seg_t0, const int* entry_first_seg,
                                 int n_segments, float* w_rows, float* u_rows, float* cum, float* k_rows, float* q_rows,
                                 float* seg_decay, float* scores, float* seg_start, float* out, int heads, int kv_heads, int dim, int vdim, cudaStream_t stream) {
  if (n_entries <= 0) return 0;
  if (heads < 1 || kv_heads < 1 || heads % kv_heads || dim < 1 || dim > segscan::MAX_DIM || vdim < 1 || heads > 65535 || n_entries > 65535)
    return IFX_ERR_UNSUPPORTED;
  GdArgs p{qkv, stride, q_col, k_col, v_col, raw, raw_stride, a_col, b_col, dec, dec_stride, a_log, dt_bias, state, entry_q_start,
           entry_q_len, entry_slot, seg_entry, seg_t0, entry_first_seg, heads, kv_heads, dim, vdim, 0, w_rows, u_rows, cum, k_rows,
           q_rows, seg_decay, scores, out};
  p.vec = !((dim | vdim | q_col | k_col | v_col) & 3) && !(stride & 3) &&
          !(((uintptr_t)qkv | (uintptr_t)w_rows | (uintptr_t)u_rows | (uintptr_t)seg_start | (uintptr_t)k_rows | (uintptr_t)q_rows) & 15);
  int rc;
  if (n_segments <= 0) {
    const dim3 grid(heads, n_entries, (vdim + 31) / 32);
    auto kern = dec ? (dim <= 32 ? gated_delta_step_kernel<4, true> : dim <= 64 ? gated_delta_step_kernel<8, true>
                       : dim <= 128 ? gated_delta_step_kernel<16, true> : gated_delta_step_kernel<32, true>)
                    : (dim <= 32 ? gated_delta_step_kernel<4, false> : dim <= 64 ? gated_delta_step_kernel<8, false>
                       : dim <= 128 ? gated_delta_step_kernel<16, false> : gated_delta_step_kernel<32, false>);
    rc = launch_pdl(kern, grid, dim3(256), 0, stream, p);
    return rc ? rc : IFX_LAUNCH_CHECK();
  }
  if (!w_rows || !u_rows || !seg_start) return IFX_ERR_UNSUPPORTED;
  if (dec ? !k_rows || !q_rows || !seg_decay || !scores || ((uintptr_t)scores & 15) : !cum) return IFX_ERR_UNSUPPORTED;
  {
    auto kern = dec ? channel_delta_segments_kernel : gated_delta_segments_kernel;
    const size_t smem = dec ? channel_segments_smem(dim) : segments_smem(dim);
    rc = segscan::allow_smem(kern, smem);
    if (rc) return rc;
    rc = launch_pdl(kern, dim3(n_segments, heads), dim3(THREADS), smem, stream, p);
    if (rc) return rc;
  }
  segscan::Args a{};
  a.q = qkv + q_col; a.k = qkv + k_col; a.qk_stride = stride; a.share = heads / kv_heads; a.k_scale = 1.0f;
  a.v = u_rows; a.v_stride = (long long)heads * vdim;
  a.cum = cum; a.w_rows = w_rows; a.u_rows = u_rows; a.state = state;
  a.entry_q_start = entry_q_start; a.entry_q_len = entry_q_len; a.entry_slot = entry_slot;
  a.seg_entry = seg_entry; a.seg_t0 = seg_t0; a.entry_first_seg = entry_first_seg;
  a.seg_start = seg_start; a.out = out; a.heads = heads; a.dim = dim; a.vdim = vdim;
  a.vec = p.vec && !((uintptr_t)out & 15);
  if (dec) {
    a.q = q_rows; a.k = k_rows; a.qk_stride = (long long)heads * dim; a.share = 1;
    a.seg_decay = seg_decay; a.scores = scores;
    rc = segscan::launch<false, true, true>(a, n_entries, n_segments, stream);
    return rc ? rc : IFX_LAUNCH_CHECK();
  }
  rc = segscan::launch<false, true>(a, n_entries, n_segments, stream);
  return rc ? rc : IFX_LAUNCH_CHECK();
}

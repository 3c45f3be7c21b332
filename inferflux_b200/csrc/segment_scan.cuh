// A linear-attention state over time, S_t = g_t S_{t-1} + k_t u_t^T and o_t = S_t^T q_t per head (S [dim x vdim], float32),
// for portions of prompts, cut into segments of SEG tokens.  With G_i the product of a segment's decays up to token i,
// and S the state the segment starts from,
//
//   o_i   = G_i S^T q_i + sum_{j <= i} (G_i / G_j) (q_i . k_j) u_j        tokens of a segment: one kernel over all segments
//   S_end = G_n S + sum_j (G_n / G_j) k_j u_j^T                           segment after segment: one kernel that carries S
//
// Three mixers share the two kernels below.  Where the decay is one number per head (FIXED) its powers come as a table and
// u is the value itself.  Otherwise the decays come as running sums of logarithms from the segment's start, and with
// SOLVE u = U - W S, with U and W worked out beforehand for all segments at once.  Where there is a decay per key channel
// (CHANNEL, with SOLVE; G_i is then a diagonal) all that meets it has been worked out beforehand too: the keys come times
// what is left of them at the segment's end, the queries times G_i, the scores (G_i / G_j) (q_i . k_j) as a table of their
// own, and G_n row by row.
//
// The carry: a block a (head, entry, VC value columns).  256 threads own the state in registers, a thread four
// neighbouring rows (every 128 of them) of VC / 8 columns; 128 more keep the copies of the next segments' rows into a
// ring in shared memory going, so the walk from segment to segment waits for no copy.  With SOLVE the state also lies in
// shared memory, column by column, for the product W S.
//
// The outputs: a block a (segment, head, VT value columns).  Queries and keys lie transposed in shared memory, so that a
// thread's 4 x 4 corner of q . k and its 4 x (VT / 32) corner of the results cost two 16-byte loads per 16 (8) multiply-adds;
// the scores' sum over dim is split over four groups of threads.
#pragma once
#include "common.cuh"

namespace segscan {
constexpr int SEG = 32;                 // tokens per segment
constexpr int COMPUTE = 256;            // threads that compute
constexpr int HELPERS = 128;            // threads that bring the next segment's rows
constexpr int MAX_DIM = 256;

struct Args {
  const float* q; const float* k; long long qk_stride;   // rows of q and of k heads: head h / share at dim times that
  const float* v; long long v_stride;                    // rows of value heads (the outputs kernel's u)
  int share;                                             // heads that read one query and key head
  float k_scale;                                         // keys count so many times
  const float* powers;                                   // FIXED: [heads][SEG + 1] powers of the head's decay
  const float* cum;                                      // else: [row][heads] running sums of ln g from the segment's start
  const float* seg_decay;                                // CHANNEL: [segments][heads][dim] G_n
  const float* scores;                                   // CHANNEL: [segments][heads][SEG j][SEG i], zero for j > i
  const float* w_rows; float* u_rows;                    // SOLVE: [row][heads * dim], [row][heads * vdim] (U in, u out)
  float* state;                                          // [slots][heads][dim][vdim]
  const int* entry_q_start; const int* entry_q_len; const int* entry_slot;
  const int* seg_entry; const int* seg_t0; const int* entry_first_seg;
  float* seg_start;                                      // [segments][heads][dim][vdim]
  float* out;                                            // [row][heads * vdim]
  int heads, dim, vdim, vec;                             // vec: every row and column block starts on a 16-byte boundary
};

__host__ __device__ __forceinline__ int pad4(int n) { return (n + 3) & ~3; }
__host__ __device__ __forceinline__ int pad16(int n) { return (n + 15) & ~15; }
// how far apart rows lie in shared memory: 16-byte aligned, neighbours in different banks
__host__ __device__ __forceinline__ int row_ld(int dim) { return pad4(dim) + 4; }

// Two float32 multiply-adds in one instruction, each rounded like fmaf
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(*reinterpret_cast<unsigned long long*>(&d))
      : "l"(*reinterpret_cast<const unsigned long long*>(&a)), "l"(*reinterpret_cast<const unsigned long long*>(&b)),
        "l"(*reinterpret_cast<const unsigned long long*>(&c)));
  return d;
}

// Two lanes (`mask` apart) hold parts of the same 2 H sums: the one with `upper` gives away the first H and keeps the
// others, the other the other way round; afterwards y[0 .. H) are the sums kept.
template <int H>
__device__ __forceinline__ void trade(float* y, bool upper, int mask) {
#pragma unroll
  for (int i = 0; i < H; ++i) {
    const float give = upper ? y[i] : y[i + H], keep = upper ? y[i + H] : y[i];
    y[i] = keep + __shfl_xor_sync(0xffffffffu, give, mask);
  }
}

// SEG rows of `width` floats (rows `stride` apart) into shared memory rows of `ld`: `fill` floats each, zeros behind the
// width and behind row n.  `threads` threads take part, this one is `t` of them (a multiple of 8 of them).
__device__ __forceinline__ void stage_rows(float* dst, int ld, int fill, const float* src, long long stride, int n, int width,
                                           int vec, int t, int threads) {
  if (vec) {                             // eight neighbouring threads walk a row
    for (int j = t >> 3; j < SEG; j += threads >> 3) {
      float* to = dst + j * ld;
      const float* from = src + (size_t)j * stride;
#pragma unroll 4
      for (int d = 4 * (t & 7); d < fill; d += 32) {
        if (j < n && d < width) cp_async_f32x4(to + d, from + d);
        else *reinterpret_cast<float4*>(to + d) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      }
    }
  } else {
    for (int j = t >> 3; j < SEG; j += threads >> 3)
      for (int d = t & 7; d < fill; d += 8) {
        if (j < n && d < width) cp_async_f32(dst + j * ld + d, src + (size_t)j * stride + d);
        else dst[j * ld + d] = 0.0f;
      }
  }
}

// floats of a buffer that hold the decays: running sums, or (CHANNEL) one number per state row
__host__ __device__ __forceinline__ int decay_floats(int dim, bool channel) { return channel ? row_ld(dim) : SEG; }
template <int VC> __host__ __device__ __forceinline__ int carry_buffer(int dim, bool solve, bool channel) {
  return SEG * row_ld(dim) + (solve ? SEG * row_ld(dim) : 0) + SEG * VC + decay_floats(dim, channel);
}
template <int VC, int NB> inline size_t carry_smem(int dim, bool solve, bool channel) {
  return ((solve ? VC * row_ld(dim) : 0) + SEG * VC + NB * (size_t)carry_buffer<VC>(dim, solve, channel)) * sizeof(float);
}

// NR: blocks of 128 state rows (1: dim up to 128, 2: up to 256).  NB: segments the ring holds.
template <bool FIXED, bool SOLVE, bool CHANNEL, int VC, int NR, int NB>
__global__ void __launch_bounds__(COMPUTE + HELPERS, 1)
carry_kernel(Args p) {
  extern __shared__ __align__(16) float sm[];
  pdl_enter();
  constexpr int NC = VC / 8;
  const int D = p.dim, V = p.vdim, DP = pad4(D), LD = row_ld(D), BUF = carry_buffer<VC>(D, SOLVE, CHANNEL), DEC = decay_floats(D, CHANNEL);
  float* us = sm;                         // [SEG][VC]: u, each times what is left of it at the segment's end
  float* St = us + SEG * VC;              // SOLVE: [VC][LD], the state's columns, rows side by side
  float* bufs = St + (SOLVE ? VC * LD : 0);            // NB of: K [SEG][LD], values [SEG][VC], decays [DEC], W [SEG][LD]
  const int h = blockIdx.x, e = blockIdx.y, v0 = blockIdx.z * VC, tid = threadIdx.x;
  const int len = p.entry_q_len[e], r0 = p.entry_q_start[e];
  const int n_seg = (len + SEG - 1) / SEG, seg0 = p.entry_first_seg[e];
  const int vcols = min(VC, V - v0);
  if (tid >= COMPUTE) {
    const int t = tid - COMPUTE;
    const float* k = p.k + (size_t)r0 * p.qk_stride + (h / p.share) * D;
    const float* v = SOLVE ? p.u_rows + ((size_t)r0 * p.heads + h) * V + v0 : p.v + (size_t)r0 * p.v_stride + h * V + v0;
    const long long vs = SOLVE ? (long long)p.heads * V : p.v_stride;
    auto stage = [&](int s) {
      float* buf = bufs + (s % NB) * BUF;
      const int t0 = s * SEG, n = min(SEG, len - t0);
      stage_rows(buf, LD, DP, k + (size_t)t0 * p.qk_stride, p.qk_stride, n, D, p.vec, t, HELPERS);
      stage_rows(buf + SEG * LD, VC, VC, v + (size_t)t0 * vs, vs, n, vcols, p.vec, t, HELPERS);
      if (CHANNEL) {
        float* c = buf + SEG * LD + SEG * VC;
        const float* g = p.seg_decay + ((size_t)(seg0 + s) * p.heads + h) * D;
        for (int d = t; d < LD; d += HELPERS) {
          if (d < D) cp_async_f32(c + d, g + d);
          else c[d] = 0.0f;
        }
      } else if (!FIXED && t < SEG) {
        float* c = buf + SEG * LD + SEG * VC + t;
        if (t < n) cp_async_f32(c, p.cum + (size_t)(r0 + t0 + t) * p.heads + h);
        else *c = 0.0f;
      }
      if (SOLVE)
        stage_rows(buf + SEG * LD + SEG * VC + DEC, LD, DP, p.w_rows + ((size_t)(r0 + t0) * p.heads + h) * D, (long long)p.heads * D, n, D,
                   p.vec, t, HELPERS);
    };
    // a group of copies a segment, empty past the last one, so that NB - 2 groups behind a segment's may be under way
    for (int s = 0; s < NB - 1; ++s) {
      if (s < n_seg) stage(s);
      cp_async_commit();
    }
    for (int s = 0; s < n_seg; ++s) {
      asm volatile("cp.async.wait_group %0;\n" ::"n"(NB - 2) : "memory");
      __syncthreads();                    // segment s is here, and s - 1, whose place the next copies take, is done with
      if (s + NB - 1 < n_seg) stage(s + NB - 1);
      cp_async_commit();
    }
    cp_async_wait_all();
    return;
  }
  const int lane = tid & 31, warp = tid >> 5;
  // Both products are bound by what a thread reads of shared memory, so a thread adds up a 4 x 4 corner of the result over
  // a part of the sum, and the lanes that hold parts of the same corner then trade until each has its own numbers whole.
  // k u^T: four rows dg .. dg + 3 (and 128 on) of four columns, every fourth token; it keeps column col (and col + 8).
  const int quad = 4 * (lane & 1), jq = (lane >> 1) & 3, col = quad + jq, dg = 4 * (4 * warp + (lane >> 3));
  // W S: four rows of four columns, every sixteenth group of four dimensions; it keeps row ur of column uc (and uc + 8).
  const int ks = lane >> 1, ur = 4 * warp + (ks >> 2), uc = quad + (ks & 3);
  int k_at[NR];
#pragma unroll
  for (int r = 0; r < NR; ++r) k_at[r] = min(128 * r + dg, DP - 4);
  float* slot = p.state + ((size_t)p.entry_slot[e] * p.heads + h) * D * V + v0;
  float S[NR][NC][4];
#pragma unroll
  for (int r = 0; r < NR; ++r)
#pragma unroll
    for (int a = 0; a < NC; ++a)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int d = 128 * r + dg + x, c = col + 8 * a;
        S[r][a][x] = (d < D && c < vcols) ? slot[(size_t)d * V + c] : 0.0f;
      }
  auto show = [&]() {                     // the state's columns for the product W S
#pragma unroll
    for (int r = 0; r < NR; ++r)
      if (128 * r + dg < DP)
#pragma unroll
        for (int a = 0; a < NC; ++a)
          *reinterpret_cast<float4*>(St + (col + 8 * a) * LD + 128 * r + dg) = make_float4(S[r][a][0], S[r][a][1], S[r][a][2], S[r][a][3]);
  };
  if (SOLVE) show();
  const float* pw = FIXED ? p.powers + h * (SEG + 1) : nullptr;
  const bool inside = vcols == VC && D == 128 * NR;                 // no thread holds a row or column that does not exist
  float* start = p.seg_start + ((size_t)seg0 * p.heads + h) * D * V + v0 + (size_t)dg * V + col;
  const size_t start_step = (size_t)p.heads * D * V;
  float* udst = SOLVE ? p.u_rows + ((size_t)(r0 + ur) * p.heads + h) * V + v0 + uc : nullptr;
  const size_t u_step = (size_t)SEG * p.heads * V;
  for (int s = 0; s < n_seg; ++s, start += start_step, udst += u_step) {
    const float* K = bufs + (s % NB) * BUF;
    const float* U = K + SEG * LD;
    const float* cs = U + SEG * VC;
    const int n = min(SEG, len - s * SEG);
    __syncthreads();                      // this segment's rows are here and the state is shown
    float total = 0.0f, left;
    if (CHANNEL) {
      left = 1.0f;
    } else if (FIXED) {
      total = pw[n];
      left = ur < n ? pw[n - 1 - ur] * p.k_scale : 0.0f;
    } else {
      const float last = cs[n - 1];
      total = expf(last);
      left = ur < n ? expf(last - cs[ur]) * p.k_scale : 0.0f;
    }
    float u[NC];
#pragma unroll
    for (int a = 0; a < NC; ++a) u[a] = U[ur * VC + uc + 8 * a];
    if (SOLVE) {
      const float* W = cs + DEC + 4 * warp * LD + 4 * ks;
      const float* X = St + quad * LD + 4 * ks;
      float2 acc[NC][16] = {};            // [row][column], even and odd dimensions apart
#pragma unroll 2
      for (int d = 0; d < DP - 4 * ks; d += 64) {
        float4 w[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) w[x] = *reinterpret_cast<const float4*>(W + x * LD + d);
#pragma unroll
        for (int a = 0; a < NC; ++a)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float4 v = *reinterpret_cast<const float4*>(X + (8 * a + c) * LD + d);
#pragma unroll
            for (int x = 0; x < 4; ++x) {
              acc[a][4 * x + c] = fma2(make_float2(w[x].x, w[x].y), make_float2(v.x, v.y), acc[a][4 * x + c]);
              acc[a][4 * x + c] = fma2(make_float2(w[x].z, w[x].w), make_float2(v.z, v.w), acc[a][4 * x + c]);
            }
          }
      }
#pragma unroll
      for (int a = 0; a < NC; ++a) {
        float y[16];
#pragma unroll
        for (int x = 0; x < 16; ++x) y[x] = acc[a][x].x + acc[a][x].y;
        trade<8>(y, ks & 8, 16);
        trade<4>(y, ks & 4, 8);
        trade<2>(y, ks & 2, 4);
        trade<1>(y, ks & 1, 2);
        u[a] -= y[0];
        if (ur < n && uc + 8 * a < vcols) udst[8 * a] = u[a];
      }
    }
#pragma unroll
    for (int a = 0; a < NC; ++a) us[ur * VC + uc + 8 * a] = ur < n ? u[a] * left : 0.0f;
#pragma unroll
    for (int r = 0; r < NR; ++r)
#pragma unroll
      for (int a = 0; a < NC; ++a)
#pragma unroll
        for (int x = 0; x < 4; ++x)
          if (inside || (128 * r + dg + x < D && col + 8 * a < vcols)) start[(size_t)(128 * r + x) * V + 8 * a] = S[r][a][x];
    asm volatile("bar.sync 1, %0;\n" ::"n"(COMPUTE) : "memory");
    if (16 * warp < DP) {                 // rows that do not exist read the last ones that do, and are never shown or stored
      float add[NR][NC][16] = {};         // [column][row]; rows behind the segment's end are zeros
      const float* kj = K + jq * LD;
      const float* uj = us + jq * VC + quad;
#pragma unroll 4
      for (int j = 0; j < SEG; j += 4, kj += 4 * LD, uj += 4 * VC) {
        float4 u4[NC];
#pragma unroll
        for (int a = 0; a < NC; ++a) u4[a] = *reinterpret_cast<const float4*>(uj + 8 * a);
#pragma unroll
        for (int r = 0; r < NR; ++r) {
          const float4 k = *reinterpret_cast<const float4*>(kj + k_at[r]);
          const float kv[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
          for (int a = 0; a < NC; ++a) {
            const float uv[4] = {u4[a].x, u4[a].y, u4[a].z, u4[a].w};
#pragma unroll
            for (int c = 0; c < 4; ++c)
#pragma unroll
              for (int x = 0; x < 4; ++x) add[r][a][4 * c + x] = fmaf(kv[x], uv[c], add[r][a][4 * c + x]);
          }
        }
      }
      // the segment's own sum is whole before it joins what is left of the state
#pragma unroll
      for (int r = 0; r < NR; ++r)
#pragma unroll
        for (int a = 0; a < NC; ++a) {
          trade<8>(add[r][a], jq & 2, 4);
          trade<4>(add[r][a], jq & 1, 2);
#pragma unroll
          for (int x = 0; x < 4; ++x) S[r][a][x] = fmaf(CHANNEL ? cs[k_at[r] + x] : total, S[r][a][x], add[r][a][x]);
        }
    }
    if (SOLVE) show();
  }
#pragma unroll
  for (int r = 0; r < NR; ++r)
#pragma unroll
    for (int a = 0; a < NC; ++a)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int d = 128 * r + dg + x, c = col + 8 * a;
        if (d < D && c < vcols) slot[(size_t)d * V + c] = S[r][a][x];
      }
}

template <int VT> inline size_t outputs_smem(int dim, bool channel) {
  const int dq = pad16(dim), kt = channel ? SEG * SEG : dq * SEG > 4 * SEG * SEG ? dq * SEG : 4 * SEG * SEG;
  return ((size_t)dq * SEG + kt + (size_t)(dq + SEG) * VT + 2 * SEG + 1) * sizeof(float);
}

// SEG rows of a head into shared memory [dq][SEG], transposed (a lane a token), zeros behind the head and behind row n
__device__ __forceinline__ void stage_transposed(float* dst, const float* src, long long stride, int n, int D, int dq, int vec, int tid) {
  const int j = tid & 31;
  const float* row = src + (size_t)j * stride;
  if (vec) {
    for (int d = 4 * (tid >> 5); d < dq; d += 4 * (COMPUTE / 32)) {
      const float4 x = (j < n && d < D) ? *reinterpret_cast<const float4*>(row + d) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
      dst[d * SEG + j] = x.x; dst[(d + 1) * SEG + j] = x.y; dst[(d + 2) * SEG + j] = x.z; dst[(d + 3) * SEG + j] = x.w;
    }
  } else {
    for (int d = tid >> 5; d < dq; d += COMPUTE / 32) dst[d * SEG + j] = (j < n && d < D) ? row[d] : 0.0f;
  }
}

template <bool FIXED, bool CHANNEL, int VT>
__global__ void __launch_bounds__(COMPUTE, 2)
outputs_kernel(Args p) {
  extern __shared__ __align__(16) float sm[];
  pdl_enter();
  constexpr int TC = VT / 32;             // columns of a thread
  const int D = p.dim, V = p.vdim, DQ = pad16(D);
  float* Qt = sm;                         // [DQ][SEG]
  float* Kt = Qt + DQ * SEG;              // [DQ][SEG], then the scores: four parts [SEG j][SEG i], then their sum in the first
  float* B = Kt + (CHANNEL ? SEG * SEG : max(DQ * SEG, 4 * SEG * SEG));        // [DQ][VT] the starting state, [SEG][VT] u
  float* lead = B + (DQ + SEG) * VT;      // [SEG] what is left of the starting state at each token
  float* dec = lead + SEG;                // [SEG + 1] powers or running sums of ln g
  const int seg = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT, tid = threadIdx.x;
  const int e = p.seg_entry[seg], t0 = p.seg_t0[seg];
  const int n = min(SEG, p.entry_q_len[e] - t0), row0 = p.entry_q_start[e] + t0;
  const int vcols = min(VT, V - v0);
  const float* start = p.seg_start + ((size_t)seg * p.heads + h) * D * V + v0;
  const float* urow = p.v + (size_t)row0 * p.v_stride + h * V + v0;
  if (p.vec) {
    for (int idx = tid; idx < (DQ + SEG) * (VT / 4); idx += COMPUTE) {
      const int d = idx / (VT / 4), c = 4 * (idx - d * (VT / 4));
      float* dst = B + d * VT + c;
      if (c < vcols && d < D) cp_async_f32x4(dst, start + (size_t)d * V + c);
      else if (c < vcols && d >= DQ && d - DQ < n) cp_async_f32x4(dst, urow + (size_t)(d - DQ) * p.v_stride + c);
      else *reinterpret_cast<float4*>(dst) = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
  } else {
    for (int idx = tid; idx < (DQ + SEG) * VT; idx += COMPUTE) {
      const int d = idx / VT, c = idx - d * VT;
      float x = 0.0f;
      if (c < vcols && d < D) x = start[(size_t)d * V + c];
      else if (c < vcols && d >= DQ && d - DQ < n) x = urow[(size_t)(d - DQ) * p.v_stride + c];
      B[idx] = x;
    }
  }
  if (CHANNEL) {                          // the scores as they are to be multiplied (always 16-byte aligned)
    const float* a = p.scores + ((size_t)seg * p.heads + h) * SEG * SEG;
    for (int idx = 4 * tid; idx < SEG * SEG; idx += 4 * COMPUTE) cp_async_f32x4(Kt + idx, a + idx);
  }
  cp_async_commit();
  const size_t qk = (size_t)row0 * p.qk_stride + (h / p.share) * D;
  stage_transposed(Qt, p.q + qk, p.qk_stride, n, D, DQ, p.vec, tid);
  if (!CHANNEL) stage_transposed(Kt, p.k + qk, p.qk_stride, n, D, DQ, p.vec, tid);
  if (CHANNEL) {
    if (tid < SEG) lead[tid] = 1.0f;
  } else if (tid < SEG) {
    if (FIXED) {
      dec[tid] = p.powers[h * (SEG + 1) + tid];
      lead[tid] = p.powers[h * (SEG + 1) + tid + 1];
    } else {
      const float c = tid < n ? p.cum[(size_t)(row0 + tid) * p.heads + h] : 0.0f;
      dec[tid] = c;
      lead[tid] = expf(c);
    }
  }
  __syncthreads();
  if (!CHANNEL) {                         // the scores, a quarter of the head's dimensions a group of 64 threads
    const int part = tid >> 6, ti = 4 * (tid & 7), tj = 4 * ((tid >> 3) & 7);
    float s[4][4] = {};
    const int per = DQ >> 2;
#pragma unroll 4
    for (int d = part * per; d < (part + 1) * per; ++d) {
      const float4 a = *reinterpret_cast<const float4*>(Qt + d * SEG + ti), b = *reinterpret_cast<const float4*>(Kt + d * SEG + tj);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) s[j][i] = fmaf(av[i], bv[j], s[j][i]);
    }
    __syncthreads();                      // the keys have been read: their place takes the parts
#pragma unroll
    for (int j = 0; j < 4; ++j)
      *reinterpret_cast<float4*>(Kt + (part * SEG + tj + j) * SEG + ti) = make_float4(s[j][0], s[j][1], s[j][2], s[j][3]);
  }
  if (!CHANNEL) __syncthreads();
  if (!CHANNEL) {                         // their sum, decayed and masked, in the first part's place (read by this thread alone)
    const int j = tid >> 3, i0 = 4 * (tid & 7);
    float v[4] = {};
#pragma unroll
    for (int part = 0; part < 4; ++part) {
      const float4 x = *reinterpret_cast<const float4*>(Kt + (part * SEG + j) * SEG + i0);
      v[0] += x.x; v[1] += x.y; v[2] += x.z; v[3] += x.w;
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int i = i0 + x;
      const float f = j > i || i >= n ? 0.0f : FIXED ? dec[max(i - j, 0)] : expf(dec[i] - dec[j]);
      v[x] = j > i || i >= n ? 0.0f : v[x] * (f * p.k_scale);
    }
    *reinterpret_cast<float4*>(Kt + j * SEG + i0) = make_float4(v[0], v[1], v[2], v[3]);
  }
  cp_async_wait_all();
  __syncthreads();
  const int ti = 4 * (tid & 7), c0 = TC * (tid >> 3);
  float acc[4][TC] = {}, own[4][TC] = {}; // from the starting state, from the segment's own tokens
  auto step = [&](float (&acc)[4][TC], const float* A, const float* b) {
    const float4 a = *reinterpret_cast<const float4*>(A);
    const float av[4] = {a.x, a.y, a.z, a.w};
    float bv[TC];
    if (TC == 4) {
      const float4 x = *reinterpret_cast<const float4*>(b);
      bv[0] = x.x; bv[1] = x.y; bv[TC - 2] = x.z; bv[TC - 1] = x.w;
    } else {
      const float2 x = *reinterpret_cast<const float2*>(b);
      bv[0] = x.x; bv[1] = x.y;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int c = 0; c < TC; ++c) acc[i][c] = fmaf(av[i], bv[c], acc[i][c]);
  };
#pragma unroll 8
  for (int d = 0; d < DQ; ++d) step(acc, Qt + d * SEG + ti, B + d * VT + c0);
#pragma unroll 8
  for (int j = 0; j < SEG; ++j) step(own, Kt + j * SEG + ti, B + (DQ + j) * VT + c0);
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int c = 0; c < TC; ++c) acc[i][c] = fmaf(lead[ti + i], acc[i][c], own[i][c]);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (ti + i >= n) continue;
    float* dst = p.out + ((size_t)(row0 + ti + i) * p.heads + h) * V + v0 + c0;
    if (p.vec && TC == 4) {
      if (c0 < vcols) *reinterpret_cast<float4*>(dst) = make_float4(acc[i][0], acc[i][1], acc[i][TC - 2], acc[i][TC - 1]);
    } else {
#pragma unroll
      for (int c = 0; c < TC; ++c)
        if (c0 + c < vcols) dst[c] = acc[i][c];
    }
  }
}

template <typename Kern> inline int allow_smem(Kern kern, size_t bytes) {
  return bytes > 48 * 1024 ? (int)cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) : 0;
}

template <bool FIXED, bool SOLVE, bool CHANNEL, int VC, int NR, int NB> int launch_carry(const Args& p, int n_entries, cudaStream_t stream) {
  const size_t smem = carry_smem<VC, NB>(p.dim, SOLVE, CHANNEL);
  const int rc = allow_smem(carry_kernel<FIXED, SOLVE, CHANNEL, VC, NR, NB>, smem);
  if (rc) return rc;
  return launch_pdl(carry_kernel<FIXED, SOLVE, CHANNEL, VC, NR, NB>, dim3(p.heads, n_entries, (p.vdim + VC - 1) / VC), dim3(COMPUTE + HELPERS), smem, stream, p);
}
template <bool FIXED, bool CHANNEL, int VT> int launch_outputs(const Args& p, int n_segments, cudaStream_t stream) {
  const size_t smem = outputs_smem<VT>(p.dim, CHANNEL);
  const int rc = allow_smem(outputs_kernel<FIXED, CHANNEL, VT>, smem);
  if (rc) return rc;
  return launch_pdl(outputs_kernel<FIXED, CHANNEL, VT>, dim3(n_segments, p.heads, (p.vdim + VT - 1) / VT), dim3(COMPUTE), smem, stream, p);
}

// Both kernels, one after the other.  Narrow column blocks where they fit the SMs at once.
template <bool FIXED, bool SOLVE, bool CHANNEL = false> int launch(const Args& p, int n_entries, int n_segments, cudaStream_t stream) {
  const bool wide = (long long)p.heads * n_entries * ((p.vdim + 7) / 8) > 148;
  int rc;
  if (p.dim <= 128)
    rc = wide ? launch_carry<FIXED, SOLVE, CHANNEL, 16, 1, 4>(p, n_entries, stream) : launch_carry<FIXED, SOLVE, CHANNEL, 8, 1, 4>(p, n_entries, stream);
  else
    rc = wide ? launch_carry<FIXED, SOLVE, CHANNEL, 16, 2, 2>(p, n_entries, stream) : launch_carry<FIXED, SOLVE, CHANNEL, 8, 2, 2>(p, n_entries, stream);
  if (rc) return rc;
  return p.vdim > 64 ? launch_outputs<FIXED, CHANNEL, 128>(p, n_segments, stream) : launch_outputs<FIXED, CHANNEL, 64>(p, n_segments, stream);
}
}  // namespace segscan

// Retention: linear attention with a fixed decay per head, no softmax and no denominator,
//
//   S_t = g S_{t-1} + k_t v_t^T          S: [dim x vdim] per head, float32, in the request's state slot
//   o_t = S_t^T q_t                      g = the head's decay, k already scaled; q, k and v through silu on the way in
//                                        where a design asks for it
//
// Portions are cut into segments of 32 tokens: the states the segments start from one after the other, then every
// segment's outputs side by side (segment_scan.cuh), with the powers of the decay as a table.  A step of single tokens has a
// kernel of its own, which streams the state through registers.  All of it is float32 FFMA: the state, what enters it
// and the scores are 32-bit by the mixer's definition.
// `finish` divides each head's output by its root mean square, multiplies by silu(gate) and rounds once.
#include "segment_scan.cuh"

namespace {
struct RetStep {
  const float* proj; int stride;       // [N][stride] float32, q and k already rotated
  int q_col, k_col, v_col;             // first column of q, k, v (heads side by side, dim / vdim wide)
  int heads, dim, vdim;
  const float* powers;                 // [heads][SEG + 1]: the decay's powers, 0 up to SEG
  float k_scale;
  int silu;                            // q, k and v are silu(projection)
  const int* entry_q_start; const int* entry_q_len; const int* entry_slot;
  float* state;                        // [slots][heads][dim][vdim]
};

__device__ __forceinline__ float taken(const RetStep& s, size_t row, int col) {
  const float x = s.proj[row * s.stride + col];
  return s.silu ? x / (1.0f + expf(-x)) : x;
}

// q, k and v columns through silu, in place (portions; single tokens take it on the way in).  N columns a thread: 4 with
// 16-byte accesses where everything is a multiple of them, else 1.
template <int N>
__global__ void __launch_bounds__(256)
retention_silu_kernel(RetStep s, float* __restrict__ proj, int width_qk, int width_v) {
  pdl_enter();
  float* row = proj + (size_t)blockIdx.x * s.stride;
  for (int i = N * threadIdx.x; i < 2 * width_qk + width_v; i += N * blockDim.x) {
    float* x = row + (i < width_qk ? s.q_col + i : i < 2 * width_qk ? s.k_col + i - width_qk : s.v_col + i - 2 * width_qk);
    if (N == 4) {
      float4 v = *reinterpret_cast<float4*>(x);
      v.x = v.x / (1.0f + expf(-v.x)); v.y = v.y / (1.0f + expf(-v.y));
      v.z = v.z / (1.0f + expf(-v.z)); v.w = v.w / (1.0f + expf(-v.w));
      *reinterpret_cast<float4*>(x) = v;
    } else {
      *x = *x / (1.0f + expf(-*x));
    }
  }
}

// Single tokens, one per entry: a block a (head, entry, 32 value columns), eight threads a column, NI state rows a thread
// in registers between the slot's read and its write.
template <int NI>
__global__ void __launch_bounds__(256)
retention_step_kernel(RetStep s, float* __restrict__ out) {
  __shared__ float ks[8 * NI], qs[8 * NI], red[8][33];
  pdl_enter();
  const int head = blockIdx.x, e = blockIdx.y, tid = threadIdx.x, lane = tid & 31, grp = tid >> 5;
  const int D = s.dim, V = s.vdim, c = blockIdx.z * 32 + lane;
  const bool on = c < V;
  const size_t row = s.entry_q_start[e];
  float* st = s.state + ((size_t)s.entry_slot[e] * s.heads + head) * D * V + (on ? c : 0);
  float S[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = grp + 8 * i;
    S[i] = (on && d < D) ? st[(size_t)d * V] : 0.0f;
  }
  for (int d = tid; d < 8 * NI; d += 256) {
    ks[d] = d < D ? taken(s, row, s.k_col + head * D + d) * s.k_scale : 0.0f;
    qs[d] = d < D ? taken(s, row, s.q_col + head * D + d) : 0.0f;
  }
  const float v = on ? taken(s, row, s.v_col + head * V + c) : 0.0f;
  const float g = s.powers[head * (segscan::SEG + 1) + 1];
  __syncthreads();
  float o = 0.0f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int d = grp + 8 * i;
    S[i] = fmaf(g, S[i], ks[d] * v);
    o = fmaf(qs[d], S[i], o);
    if (on && d < D) st[(size_t)d * V] = S[i];
  }
  red[grp][lane] = o;
  __syncthreads();
  if (grp == 0 && on) {
    o = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) o += red[w][lane];
    out[(row * s.heads + head) * V + c] = o;
  }
}

// out[t][h][:] = o[t][h][:] / sqrt(mean(o^2) + eps) * silu(gate[t][h][:]); a warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256)
retention_finish_kernel(const float* __restrict__ o, const float* __restrict__ gate, int gate_stride, T* __restrict__ out,
                        long long out_stride, int n_tokens, int heads, int vdim, float eps) {
  pdl_enter();
  const int w = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (w >= n_tokens * heads) return;
  const int t = w / heads, h = w - t * heads;
  const float* row = o + ((size_t)t * heads + h) * vdim;
  float ss = 0.0f;
  for (int d = lane; d < vdim; d += 32) ss = fmaf(row[d], row[d], ss);
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
  const float* gr = gate + (size_t)t * gate_stride + (size_t)h * vdim;
  T* orow = out + (size_t)t * out_stride + (size_t)h * vdim;
  for (int d = lane; d < vdim; d += 32) {
    const float gv = gr[d];
    orow[d] = Num<T>::from_f(row[d] * inv * (gv / (1.0f + expf(-gv))));
  }
}
}  // namespace

IFX_API int ifx_retention_segment() { return segscan::SEG; }

// proj: float32 [N][stride] with q, k (rotated) and v at the given columns, through silu first if asked for (portions: in
// place).  powers: float32 [heads][segment + 1], the head's decay to the 0th, 1st, .. power.  A step of single tokens
// (n_rows <= n_entries) needs no segments; otherwise seg_start [segments][heads][dim][vdim] float32 is scratch.
IFX_API int ifx_retention_scan(float* proj, int stride, int q_col, int k_col, int v_col, int heads, int dim, int vdim,
                               const float* powers, float k_scale, int silu, float* state,
                               const int* seg_entry, const int* seg_t0, int n_segments, const int* entry_first_seg,
                               const int* entry_q_start, const int* entry_q_len, const int* entry_slot, int n_entries,
                               int n_rows, float* seg_start, float* out, cudaStream_t stream) {
  if (n_rows <= 0 || n_entries <= 0) return 0;
  if (dim < 1 || dim > segscan::MAX_DIM || vdim < 1 || heads < 1 || heads > 65535 || n_entries > 65535) return IFX_ERR_UNSUPPORTED;
  RetStep s{proj, stride, q_col, k_col, v_col, heads, dim, vdim, powers, k_scale, silu, entry_q_start, entry_q_len, entry_slot, state};
  int rc;
  if (n_rows <= n_entries) {
    const dim3 grid(heads, n_entries, (vdim + 31) / 32);
    if (dim <= 32) rc = launch_pdl(retention_step_kernel<4>, grid, dim3(256), 0, stream, s, out);
    else if (dim <= 64) rc = launch_pdl(retention_step_kernel<8>, grid, dim3(256), 0, stream, s, out);
    else if (dim <= 128) rc = launch_pdl(retention_step_kernel<16>, grid, dim3(256), 0, stream, s, out);
    else rc = launch_pdl(retention_step_kernel<32>, grid, dim3(256), 0, stream, s, out);
    return rc ? rc : IFX_LAUNCH_CHECK();
  }
  if (!seg_start || n_segments <= 0) return IFX_ERR_UNSUPPORTED;
  segscan::Args a{};
  a.q = proj + q_col; a.k = proj + k_col; a.qk_stride = stride; a.share = 1; a.k_scale = k_scale;
  a.v = proj + v_col; a.v_stride = stride; a.powers = powers; a.state = state;
  a.entry_q_start = entry_q_start; a.entry_q_len = entry_q_len; a.entry_slot = entry_slot;
  a.seg_entry = seg_entry; a.seg_t0 = seg_t0; a.entry_first_seg = entry_first_seg;
  a.seg_start = seg_start; a.out = out; a.heads = heads; a.dim = dim; a.vdim = vdim;
  a.vec = !((dim | vdim | q_col | k_col | v_col | stride) & 3) && !(((uintptr_t)proj | (uintptr_t)seg_start | (uintptr_t)out) & 15);
  if (silu) {
    rc = a.vec ? launch_pdl(retention_silu_kernel<4>, dim3(n_rows), dim3(256), 0, stream, s, proj, heads * dim, heads * vdim)
               : launch_pdl(retention_silu_kernel<1>, dim3(n_rows), dim3(256), 0, stream, s, proj, heads * dim, heads * vdim);
    if (rc) return rc;
  }
  rc = segscan::launch<true, false>(a, n_entries, n_segments, stream);
  return rc ? rc : IFX_LAUNCH_CHECK();
}

IFX_API int ifx_retention_finish(const float* o, const float* gate, int gate_stride, void* out, int out_dtype,
                                 long long out_stride, int n_tokens, int heads, int vdim, float eps, cudaStream_t stream) {
  const int warps = n_tokens * heads;
  if (warps <= 0) return 0;
  const dim3 grid((warps + 7) / 8);
  const int rc = out_dtype == IFX_BF16
      ? launch_pdl(retention_finish_kernel<bf16>, grid, dim3(256), 0, stream, o, gate, gate_stride, (bf16*)out, out_stride, n_tokens, heads, vdim, eps)
      : launch_pdl(retention_finish_kernel<float>, grid, dim3(256), 0, stream, o, gate, gate_stride, (float*)out, out_stride, n_tokens, heads, vdim, eps);
  return rc ? rc : IFX_LAUNCH_CHECK();
}

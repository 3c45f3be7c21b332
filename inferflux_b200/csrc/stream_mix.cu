// A residual stream of S copies, X float32 [N][S][hidden] (S up to 16):
//
//   stream_mix_norm   X_t <- sum_s mix[s][t] X_s + w_out[t] * (y_0 + y_1 + ...)      all copies at once from the old ones
//                     u = sum_s reads[s] X_s;   out = u / sqrt(mean(u^2) + eps) * weight
//   embed_bigram      x = E[id] + B[(previous * mul_prev + id * mul_cur) mod buckets], written to every copy
//
// stream_mix_norm is one pass over the row: a sublayer's pending result is mixed in, the sum that the next sublayer reads
// is taken from the new copies while they are still in registers, and its norm follows from shared memory.  One block
// per output row; source row = rows ? rows[blockIdx.x] : blockIdx.x, and in that gather mode the copies are left as they
// are in memory.  The order of additions depends on the row's length alone.
//
// embed_bigram reads the token ahead of an entry's first one from the request's slot (stored one up: 0 = there is none,
// and the row behind the hashed ones is taken) and leaves the entry's last token there; the block of the entry's first
// row does both, so no other block depends on the slot.
#include "common.cuh"

namespace {
constexpr int MAX_STREAMS = 16;

struct StreamArgs {
  float* x; const float* mix; const float* w_out; const float* reads; const float* weight; const int* rows;
  long long part_stride; int parts; int hidden; int streams; int write; float eps;
};

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
  const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<unsigned*>(&a);
  u.y = *reinterpret_cast<unsigned*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

// V: one number or four neighbouring ones
template <int W> struct Vec;
template <> struct Vec<1> {
  float v[1];
  template <typename T> static __device__ __forceinline__ Vec load(const T* p) { return Vec{{Num<T>::to_f(*p)}}; }
  template <typename T> __device__ __forceinline__ void store(T* p) const { *p = Num<T>::from_f(v[0]); }
};
template <> struct Vec<4> {
  float v[4];
  template <typename T> static __device__ __forceinline__ Vec load(const T* p) {
    const float4 a = load4(p);
    return Vec{{a.x, a.y, a.z, a.w}};
  }
  template <typename T> __device__ __forceinline__ void store(T* p) const { store4(p, make_float4(v[0], v[1], v[2], v[3])); }
};

// S: the number of copies, or 0 for any number up to MAX_STREAMS.  W: columns a thread takes at a time.
template <int S, int W, typename TY, typename TO>
__global__ void __launch_bounds__(512, 2)
stream_mix_norm_kernel(StreamArgs p, const TY* __restrict__ y, TO* __restrict__ out) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float u_buf[];            // [hidden]
  __shared__ float scratch[32];
  constexpr int SM = S ? S : MAX_STREAMS;
  const int ns = S ? S : p.streams, hidden = p.hidden;
  // volatile, in shared memory: kept in registers these would halve the occupancy.  They are parameters, so they are
  // read before the kernel ahead has finished.
  __shared__ volatile float reads[SM], w_out[SM], mix[SM * SM];
  for (int i = threadIdx.x; i < ns * ns; i += blockDim.x) {
    if (i < ns) {
      reads[i] = p.reads[i];
      if (y) w_out[i] = p.w_out[i];
    }
    if (y) mix[i] = p.mix[i];
  }
  __syncthreads();
  pdl_wait();
  const int src = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  float* xr = p.x + (size_t)src * ns * hidden;
  const TY* yr = y ? y + (size_t)src * hidden : nullptr;
  float ss = 0.0f;
#pragma unroll 1
  for (int i = W * threadIdx.x; i < hidden; i += W * blockDim.x) {
    Vec<W> x[SM], u;
#pragma unroll
    for (int s = 0; s < SM; ++s)
      if (s < ns) x[s] = Vec<W>::load(xr + (size_t)s * hidden + i);
#pragma unroll
    for (int c = 0; c < W; ++c) u.v[c] = 0.0f;
    if (yr) {
      Vec<W> d = Vec<W>::load(yr + i);
      for (int q = 1; q < p.parts; ++q) {
        const Vec<W> more = Vec<W>::load(yr + (size_t)q * p.part_stride + i);
#pragma unroll
        for (int c = 0; c < W; ++c) d.v[c] += more.v[c];
      }
#pragma unroll (S ? S : 1)
      for (int t = 0; t < SM; ++t) {
        if (t >= ns) break;
        Vec<W> a;
#pragma unroll
        for (int c = 0; c < W; ++c) a.v[c] = w_out[t] * d.v[c];
#pragma unroll
        for (int s = 0; s < SM; ++s) {
          if (s >= ns) break;
          const float m = mix[s * ns + t];
#pragma unroll
          for (int c = 0; c < W; ++c) a.v[c] = fmaf(m, x[s].v[c], a.v[c]);
        }
        if (p.write) a.store(xr + (size_t)t * hidden + i);
#pragma unroll
        for (int c = 0; c < W; ++c) u.v[c] = fmaf(reads[t], a.v[c], u.v[c]);
      }
    } else {
#pragma unroll
      for (int s = 0; s < SM; ++s) {
        if (s >= ns) break;
#pragma unroll
        for (int c = 0; c < W; ++c) u.v[c] = fmaf(reads[s], x[s].v[c], u.v[c]);
      }
    }
#pragma unroll
    for (int c = 0; c < W; ++c) ss = fmaf(u.v[c], u.v[c], ss);
    u.store(u_buf + i);
  }
  ss = block_sum(ss, scratch);
  const float r = 1.0f / sqrtf(ss / (float)hidden + p.eps);
  TO* o = out + (size_t)blockIdx.x * hidden;
  for (int i = W * threadIdx.x; i < hidden; i += W * blockDim.x) {      // each thread reads back what it wrote
    Vec<W> u = Vec<W>::load(u_buf + i);
    const Vec<W> w = Vec<W>::load(p.weight + i);
#pragma unroll
    for (int c = 0; c < W; ++c) u.v[c] = u.v[c] * r * w.v[c];
    u.store(o + i);
  }
}

template <int S, int W, typename TY, typename TO>
int launch_mix(const StreamArgs& p, const void* y, void* out, int n_rows, cudaStream_t stream) {
  const size_t smem = (size_t)p.hidden * sizeof(float);
  auto kern = stream_mix_norm_kernel<S, W, TY, TO>;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  const int per = (p.hidden + W - 1) / W;
  const int threads = per >= 512 ? 512 : per >= 256 ? 256 : per >= 128 ? 128 : 64;
  return launch_pdl(kern, dim3(n_rows), dim3(threads), smem, stream, p, (const TY*)y, (TO*)out);
}
template <int S, int W, typename TY>
int launch_mix_out(const StreamArgs& p, const void* y, void* out, int out_dtype, int n_rows, cudaStream_t stream) {
  return out_dtype == IFX_BF16 ? launch_mix<S, W, TY, bf16>(p, y, out, n_rows, stream) : launch_mix<S, W, TY, float>(p, y, out, n_rows, stream);
}
template <int S>
int launch_mix_types(const StreamArgs& p, const void* y, int y_dtype, void* out, int out_dtype, int vec, int n_rows, cudaStream_t stream) {
  constexpr int W = S ? 4 : 1;             // many copies leave no registers for four columns
  if (y_dtype == IFX_BF16)
    return vec ? launch_mix_out<S, W, bf16>(p, y, out, out_dtype, n_rows, stream) : launch_mix_out<S, 1, bf16>(p, y, out, out_dtype, n_rows, stream);
  return vec ? launch_mix_out<S, W, float>(p, y, out, out_dtype, n_rows, stream) : launch_mix_out<S, 1, float>(p, y, out, out_dtype, n_rows, stream);
}

struct BigramArgs {
  const int* ids; int* last; const int* row_entry; const int* entry_q_start; const int* entry_q_len; const int* entry_slot;
  float* out; long long buckets, mul_prev, mul_cur; int hidden, vocab, streams, hashed;
};

template <int W, typename T>
__global__ void embed_bigram_kernel(BigramArgs p, const T* __restrict__ table, const T* __restrict__ pairs) {
  pdl_enter();
  const int r = blockIdx.x;
  const int id = p.ids[r];
  const bool ok = id >= 0 && id < p.vocab;                   // never read outside the tables
  __shared__ long long pair_row;
  if (p.hashed && threadIdx.x == 0) {
    const int e = p.row_entry[r], q0 = p.entry_q_start[e];
    long long prev = -1;
    if (r > q0) {
      prev = p.ids[r - 1];
    } else {
      int* slot = p.last + p.entry_slot[e];
      prev = (long long)*slot - 1;
      *slot = p.ids[q0 + p.entry_q_len[e] - 1] + 1;
    }
    pair_row = prev < 0 ? p.buckets : (prev * p.mul_prev + (long long)max(id, 0) * p.mul_cur) % p.buckets;
  }
  __syncthreads();
  const T* a = table + (size_t)(ok ? id : 0) * p.hidden;
  const T* b = p.hashed ? pairs + (size_t)pair_row * p.hidden : nullptr;
  float* o = p.out + (size_t)r * p.streams * p.hidden;
  for (int i = W * threadIdx.x; i < p.hidden; i += W * blockDim.x) {
    Vec<W> v = Vec<W>::load(a + i);
    if (b) {
      const Vec<W> w = Vec<W>::load(b + i);
#pragma unroll
      for (int c = 0; c < W; ++c) v.v[c] += w.v[c];
    }
#pragma unroll
    for (int c = 0; c < W; ++c) v.v[c] = ok ? v.v[c] : 0.0f;
    for (int s = 0; s < p.streams; ++s) v.store(o + (size_t)s * p.hidden + i);
  }
}
}  // namespace

IFX_API int ifx_max_streams() { return MAX_STREAMS; }

// x float32 [N][streams][hidden]; y (or null: nothing is pending) [N][hidden] in `parts` slices part_stride apart; mix
// [streams][streams] (from, to), w_out and reads [streams], weight [hidden]: float32.  write: the mixed copies go back.
IFX_API int ifx_stream_mix_norm(float* x, const void* y, int y_dtype, int parts, long long part_stride, const float* mix,
                                const float* w_out, const float* reads, const float* weight, float eps, void* out, int out_dtype,
                                const int* rows, int n_rows, int hidden, int streams, int write, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (streams < 1 || streams > MAX_STREAMS || hidden < 1 || (size_t)hidden * sizeof(float) > 200 * 1024 || (y && (!mix || !w_out || parts < 1)))
    return IFX_ERR_UNSUPPORTED;
  if ((y && y_dtype != IFX_F32 && y_dtype != IFX_BF16) || (out_dtype != IFX_F32 && out_dtype != IFX_BF16)) return IFX_ERR_UNSUPPORTED;
  const StreamArgs p{x, mix, w_out, reads, weight, rows, part_stride, parts, hidden, streams, write, eps};
  const int vec = !((hidden | part_stride) & 3) && !(((uintptr_t)x | (uintptr_t)y | (uintptr_t)weight | (uintptr_t)out) & 15);
  const int yd = y ? y_dtype : IFX_F32;
  int rc;
  switch (streams) {
    case 1: rc = launch_mix_types<1>(p, y, yd, out, out_dtype, vec, n_rows, stream); break;
    case 2: rc = launch_mix_types<2>(p, y, yd, out, out_dtype, vec, n_rows, stream); break;
    case 3: rc = launch_mix_types<3>(p, y, yd, out, out_dtype, vec, n_rows, stream); break;
    case 4: rc = launch_mix_types<4>(p, y, yd, out, out_dtype, vec, n_rows, stream); break;
    default: rc = launch_mix_types<0>(p, y, yd, out, out_dtype, vec, n_rows, stream); break;
  }
  return rc ? rc : IFX_LAUNCH_CHECK();
}

// table [vocab][hidden] and pairs [buckets + 1][hidden] (or null) of one type; last int32 [slots]; out float32
// [N][streams][hidden].
IFX_API int ifx_embed_bigram(const void* table, const void* pairs, int dtype, long long buckets, long long mul_prev, long long mul_cur,
                             const int* ids, int* last, const int* row_entry, const int* entry_q_start, const int* entry_q_len,
                             const int* entry_slot, float* out, int n_tokens, int hidden, int vocab, int streams, cudaStream_t stream) {
  if (n_tokens <= 0) return 0;
  if (streams < 1 || hidden < 1 || (pairs && (buckets < 1 || !last))) return IFX_ERR_UNSUPPORTED;
  const BigramArgs p{ids, last, row_entry, entry_q_start, entry_q_len, entry_slot, out, buckets, mul_prev, mul_cur, hidden, vocab,
                     streams, pairs != nullptr};
  const int vec = !(hidden & 3) && !(((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)out) & 15);
  const int per = vec ? hidden / 4 : hidden;
  const dim3 grid(n_tokens), block(per >= 256 ? 256 : per >= 128 ? 128 : 64);
  int rc;
  if (dtype == IFX_BF16)
    rc = vec ? launch_pdl(embed_bigram_kernel<4, bf16>, grid, block, 0, stream, p, (const bf16*)table, (const bf16*)pairs)
             : launch_pdl(embed_bigram_kernel<1, bf16>, grid, block, 0, stream, p, (const bf16*)table, (const bf16*)pairs);
  else if (dtype == IFX_F32)
    rc = vec ? launch_pdl(embed_bigram_kernel<4, float>, grid, block, 0, stream, p, (const float*)table, (const float*)pairs)
             : launch_pdl(embed_bigram_kernel<1, float>, grid, block, 0, stream, p, (const float*)table, (const float*)pairs);
  else
    return IFX_ERR_UNSUPPORTED;
  return rc ? rc : IFX_LAUNCH_CHECK();
}

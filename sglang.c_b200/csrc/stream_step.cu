// Several residual streams side by side (hyper-connections).  A token's stream rows X_0 .. X_(S-1)
// (32-bit, E wide) lie together; a sublayer reads one combination of them and its result y goes back into
// all of them.  Between two sublayers one launch does, for every token, all streams at once from the old
// ones,
//   X_t <- sum_s mix[s][t] X_s + out[t] y               (the write of the sublayer before: optional)
//   u = sum_s in[s] X_s                                  (what the next sublayer is made from)
//   h = u / sqrt(mean(u^2) + eps) * gain                 (its RMS norm; without a gain h = u)
// so a stream's row is read once and written once per sublayer.  The old rows may all be one row (stream
// stride 0: the copies that a model starts from, before anything was written).
//
// A block a row; a thread owns the same columns of every stream, so the rows may be rewritten in place,
// and the order of a row's additions depends on its width only.
#include "common.cuh"

SGLC_DEFINE_ERROR_STRING()

constexpr int STREAMS_MAX = 32;
constexpr int STREAM_THREADS = 256;

struct StreamArgs {
  const float* src; long long src_row, src_stream;   // old rows: element strides between tokens and streams
  float* dst; long long dst_row, dst_stream;         // new rows (null: nothing is written back)
  const float* y; long long y_row;                   // the sublayer's result (null: no write)
  const float* w_out; const float* w_mix;            // [S], [S][S] (from, to)
  const float* w_in;                                 // [S]
  const float* gain; float eps;
  long long h_row;
  const int* rows;                                   // null, or the rows to work on (read and written at these places)
  int n_rows, S, E, max_row;
  int* err;
};

__device__ __forceinline__ void axpy(float& a, float w, float v) { a = fmaf(w, v, a); }
__device__ __forceinline__ void axpy(float4& a, float w, const float4& v) {
  a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
}
__device__ __forceinline__ float times(float w, float v) { return w * v; }
__device__ __forceinline__ float4 times(float w, const float4& v) { return make_float4(w * v.x, w * v.y, w * v.z, w * v.w); }
__device__ __forceinline__ float squares(float v, float q) { return fmaf(v, v, q); }
__device__ __forceinline__ float squares(const float4& v, float q) {
  q = fmaf(v.x, v.x, q); q = fmaf(v.y, v.y, q); q = fmaf(v.z, v.z, q);
  return fmaf(v.w, v.w, q);
}
__device__ __forceinline__ void put(float* p, int i, float v) { p[i] = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, int i, float v) { p[i] = __float2bfloat16_rn(v); }
__device__ __forceinline__ void put(float* p, int i, const float4& v) { reinterpret_cast<float4*>(p)[i] = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, int i, const float4& v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  reinterpret_cast<uint2*>(p)[i] = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}
__device__ __forceinline__ float normed(float v, float inv, const float* gain, int i) { return v * inv * gain[i]; }
__device__ __forceinline__ float4 normed(const float4& v, float inv, const float* gain, int i) {
  const float4 g = reinterpret_cast<const float4*>(gain)[i];
  return make_float4(v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z, v.w * inv * g.w);
}

// NS streams are kept in registers; EXACT: there are NS of them, else at most so many.  TV: float or float4.
template <int NS, bool EXACT, typename TV, typename TO>
__global__ void __launch_bounds__(STREAM_THREADS, NS <= 4 ? 4 : 1)
stream_step_kernel(const StreamArgs p, TO* __restrict__ h) {
  extern __shared__ __align__(16) float srow[];      // u of this row
  __shared__ float red[33];
  __shared__ float wm[STREAMS_MAX * STREAMS_MAX], wo[STREAMS_MAX], wi[STREAMS_MAX];
  const int S = EXACT ? NS : p.S;
  pdl_launch_dependents();
  // (the weights and the row numbers are nothing that a kernel of the step writes)
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    wi[i] = p.w_in[i];
    if (p.y) wo[i] = p.w_out[i];
  }
  if (p.y)
    for (int i = threadIdx.x; i < S * S; i += blockDim.x) wm[i] = p.w_mix[i];
  const long long row = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  if (p.rows && !sglc_index_ok(row, p.max_row, p.err)) return;
  __syncthreads();
  pdl_wait();
  const int n_it = p.E / (int)(sizeof(TV) / 4);
  const TV* src = reinterpret_cast<const TV*>(p.src + row * p.src_row);
  const long long ss = p.src_stream / (long long)(sizeof(TV) / 4), ds = p.dst_stream / (long long)(sizeof(TV) / 4);
  TV* dst = p.dst ? reinterpret_cast<TV*>(p.dst + row * p.dst_row) : nullptr;
  const TV* yr = p.y ? reinterpret_cast<const TV*>(p.y + row * p.y_row) : nullptr;
  TV* su = reinterpret_cast<TV*>(srow);
  float q = 0.0f;
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    TV X[NS];
#pragma unroll
    for (int s = 0; s < NS; s++)
      if (EXACT || s < S) X[s] = src[s * ss + i];
    TV u;
    if (yr) {
      const TV yv = yr[i];
#pragma unroll(NS <= 8 ? NS : 1)
      for (int t = 0; t < NS; t++) {
        if (EXACT || t < S) {
          TV a = times(wo[t], yv);
#pragma unroll
          for (int s = 0; s < NS; s++)
            if (EXACT || s < S) axpy(a, wm[s * S + t], X[s]);
          if (dst) dst[t * ds + i] = a;
          if (t == 0) u = times(wi[0], a);
          else axpy(u, wi[t], a);
        }
      }
    } else {
      u = times(wi[0], X[0]);
#pragma unroll
      for (int s = 1; s < NS; s++)
        if (EXACT || s < S) axpy(u, wi[s], X[s]);
    }
    su[i] = u;
    q = squares(u, q);
  }
  TO* hr = h + row * p.h_row;
  if (!p.gain) {                                     // (a thread reads the columns it wrote)
    for (int i = threadIdx.x; i < n_it; i += blockDim.x) put(hr, i, su[i]);
    return;
  }
  const float inv = 1.0f / sqrtf(block_sum(q, red) / (float)p.E + p.eps);
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) put(hr, i, normed(su[i], inv, p.gain, i));
}

template <typename TV, typename TO>
static int stream_step_go(const StreamArgs& p, TO* h, int threads, size_t smem, cudaStream_t stream) {
#define GO(NS, EXACT)                                                                                            \
  do {                                                                                                           \
    if (smem > 40 * 1024)                                                                                        \
      cudaFuncSetAttribute(stream_step_kernel<NS, EXACT, TV, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize,   \
                           (int)smem);                                                                           \
    return sglc_launch(stream_step_kernel<NS, EXACT, TV, TO>, dim3(p.n_rows), dim3(threads), smem, stream, 1, true, p, h); \
  } while (0)
  switch (p.S) {
    case 1: GO(1, true);
    case 2: GO(2, true);
    case 3: GO(3, true);
    case 4: GO(4, true);
  }
  if (p.S <= 8) GO(8, false);
  GO(STREAMS_MAX, false);
#undef GO
}

static inline bool al(const void* q, uintptr_t n) { return (reinterpret_cast<uintptr_t>(q) & (n - 1)) == 0; }

// src, dst: float [..][S][E] with free strides between tokens and streams (all multiples of 4 for the
// 16-byte form); y: float rows; h: rows of h_dtype (SGLC_F32 or SGLC_BF16).  rows: null, or n_rows row
// numbers below max_row; src, y, dst and h are then all indexed by them.
SGLC_API int sglc_stream_step(const float* src, long long src_row, long long src_stream, float* dst, long long dst_row,
                              long long dst_stream, const float* y, long long y_row, const float* w_out,
                              const float* w_mix, const float* w_in, const float* gain, float eps, void* h,
                              long long h_row, int h_dtype, const int* rows, int n_rows, int max_row, int S, int E,
                              int* err, cudaStream_t stream) {
  if (n_rows <= 0) return SGLC_OK;
  if (S < 1 || E <= 0 || !src || !w_in || !h || (y && (!w_out || !w_mix)) || (dst && !y)) return SGLC_ERR_ARGUMENT;
  if (h_dtype != SGLC_F32 && h_dtype != SGLC_BF16) return SGLC_ERR_ARGUMENT;
  const size_t smem = (size_t)E * sizeof(float);
  if (S > STREAMS_MAX || smem > 200 * 1024) return SGLC_ERR_UNSUPPORTED;
  StreamArgs p = {src, src_row, src_stream, dst, dst_row, dst_stream, y, y_row, w_out, w_mix, w_in, gain, eps, h_row, rows,
                  n_rows, S, E, max_row, err};
  const bool vec = E % 4 == 0 && (src_row | src_stream | dst_row | dst_stream | y_row | h_row) % 4 == 0 && al(src, 16) &&
                   al(dst, 16) && al(y, 16) && al(gain, 16) && al(h, h_dtype == SGLC_F32 ? 16 : 8);
  const int work = vec ? E / 4 : E;
  int threads = (work + 31) / 32 * 32;
  if (threads > STREAM_THREADS) threads = STREAM_THREADS;
  if (vec) {
    if (h_dtype == SGLC_BF16) return stream_step_go<float4>(p, (__nv_bfloat16*)h, threads, smem, stream);
    return stream_step_go<float4>(p, (float*)h, threads, smem, stream);
  }
  if (h_dtype == SGLC_BF16) return stream_step_go<float>(p, (__nv_bfloat16*)h, threads, smem, stream);
  return stream_step_go<float>(p, (float*)h, threads, smem, stream);
}

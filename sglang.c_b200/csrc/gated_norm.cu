// The output stage of a recurrent mixer, for the rows of a step: a row of `width` values (one
// head's read-out, or all heads' side by side) is divided by its root mean square,
//   y = o / sqrt(mean(o^2) + eps) * gain * act(gate),
// with a gain of `width` entries that every row of a token shares and a gate of the row's shape
// taken through silu or a sigmoid (or no gate: the norm alone).  Statistics and the gate are 32-bit; the result is written in
// the precision of the product that follows.  A warp a row.
// The general form adds: rows that lie `o_pitch` apart in o (a head's read-out followed by columns
// that are not part of it); a gain of groups x width entries (every row its own); and a divisor per
// row, formed from one more column behind the row and a running maximum m per (token, row):
//   o <- o / (max(|o[width]|, exp(-m)) + 1e-6)      (the read-out of a matrix memory whose state is
//   kept times exp(-m): o[width] is the normaliser's read-out n . q)
// ahead of the norm.
// A second form (gate_then_norm_kernel) takes the gate first: with x = o * act(gate),
//   y = x / sqrt(mean(x^2) + eps) * gain
// over `groups` equal parts of a token's row, each with its own statistics and its own part of the gain.
#include "common.cuh"

SGLC_DEFINE_ERROR_STRING()

enum { GN_SILU = 0, GN_SIGMOID = 1, GN_NONE = 2 };   // GN_NONE: no gate at all (gate may be null)

template <typename TO>
__global__ void __launch_bounds__(128)
gated_norm_kernel(const float* __restrict__ o, long long o_stride, const float* __restrict__ gate,
                  long long gate_stride, const float* __restrict__ gain, TO* __restrict__ y, long long y_stride,
                  long long n_rows, int groups, int width, float eps, int act, int o_pitch, int gain_rows,
                  const float* __restrict__ m_run, long long m_stride) {
  pdl_launch_dependents();
  const long long row = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  pdl_wait();
  if (row >= n_rows) return;
  const long long t = row / groups;
  const int c0 = (int)(row % groups) * width;
  const float* op = o + t * o_stride + (row % groups) * o_pitch;
  const float* gp = act == GN_NONE ? nullptr : gate + t * gate_stride + c0;
  if (gain_rows) gain += c0;
  float pre = 1.0f;
  if (m_run) pre = 1.0f / (fmaxf(fabsf(op[width]), expf(-m_run[t * m_stride + row % groups])) + 1e-6f);
  float ss = 0.0f;
  for (int d = lane; d < width; d += 32) {
    const float v = op[d] * pre;
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  const float inv = pre / sqrtf(ss / (float)width + eps);
  TO* yp = y + t * y_stride + c0;
  for (int d = lane; d < width; d += 32) {
    if (act == GN_NONE) {
      yp[d] = from_f32<TO>(op[d] * inv * gain[d]);
      continue;
    }
    const float g = gp[d];
    const float s = 1.0f / (1.0f + expf(-g));
    yp[d] = from_f32<TO>(op[d] * inv * gain[d] * (act == GN_SILU ? g * s : s));
  }
}

// o, gate: float [T][groups*width] (row strides free); gain: float [width]; y: [T][groups*width]
// o_pitch: columns between the rows of a token in o (>= width; width + 1 and more with m_run);
// gain_rows != 0: gain is float [groups*width]; m_run: null, or float [T][groups] (rows m_stride apart).
SGLC_API int sglc_gated_norm_ext(const float* o, long long o_stride, const float* gate, long long gate_stride,
                                 const float* gain, void* y, long long y_stride, int y_dtype, int T, int groups,
                                 int width, float eps, int act, int o_pitch, int gain_rows, const float* m_run,
                                 long long m_stride, cudaStream_t stream) {
  if (T <= 0) return SGLC_OK;
  if (groups <= 0 || width <= 0 || act < GN_SILU || act > GN_NONE || (act != GN_NONE && !gate)) return SGLC_ERR_ARGUMENT;
  if (o_pitch < width + (m_run ? 1 : 0)) return SGLC_ERR_ARGUMENT;
  const long long n_rows = (long long)T * groups;
  const dim3 grid((unsigned)((n_rows + 3) / 4));
  if (y_dtype == SGLC_F32)
    return sglc_launch(gated_norm_kernel<float>, grid, dim3(128), 0, stream, 1, true, o, o_stride, gate, gate_stride,
                       gain, (float*)y, y_stride, n_rows, groups, width, eps, act, o_pitch, gain_rows, m_run, m_stride);
  if (y_dtype == SGLC_BF16)
    return sglc_launch(gated_norm_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, 1, true, o, o_stride, gate,
                       gate_stride, gain, (__nv_bfloat16*)y, y_stride, n_rows, groups, width, eps, act, o_pitch, gain_rows,
                       m_run, m_stride);
  return SGLC_ERR_ARGUMENT;
}

SGLC_API int sglc_gated_norm(const float* o, long long o_stride, const float* gate, long long gate_stride,
                             const float* gain, void* y, long long y_stride, int y_dtype, int T, int groups,
                             int width, float eps, int act, cudaStream_t stream) {
  return sglc_gated_norm_ext(o, o_stride, gate, gate_stride, gain, y, y_stride, y_dtype, T, groups, width, eps, act,
                             width, 0, nullptr, 0, stream);
}

// A block a part of a row: x is formed once and kept in shared memory.  VEC: four columns a thread.
template <typename TO, bool VEC>
__global__ void gate_then_norm_kernel(const float* __restrict__ o, long long o_stride, const float* __restrict__ gate,
                                      long long gate_stride, const float* __restrict__ gain, TO* __restrict__ y,
                                      long long y_stride, int groups, int width, float eps, int act) {
  extern __shared__ __align__(16) float xs[];
  __shared__ float red[33];
  pdl_launch_dependents();
  const long long t = blockIdx.x / groups;
  const int c0 = (int)(blockIdx.x % groups) * width;
  const float* op = o + t * o_stride + c0;
  const float* gp = gate + t * gate_stride + c0;
  auto gated = [&](float v, float g) {
    const float s = 1.0f / (1.0f + expf(-g));
    return v * (act == GN_SILU ? g * s : s);
  };
  const int n_it = VEC ? width / 4 : width;
  pdl_wait();
  float ss = 0.0f;
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    if constexpr (VEC) {
      const float4 v = reinterpret_cast<const float4*>(op)[i], g = reinterpret_cast<const float4*>(gp)[i];
      const float4 x = make_float4(gated(v.x, g.x), gated(v.y, g.y), gated(v.z, g.z), gated(v.w, g.w));
      reinterpret_cast<float4*>(xs)[i] = x;
      ss = fmaf(x.x, x.x, ss); ss = fmaf(x.y, x.y, ss); ss = fmaf(x.z, x.z, ss); ss = fmaf(x.w, x.w, ss);
    } else {
      const float x = gated(op[i], gp[i]);
      xs[i] = x;
      ss = fmaf(x, x, ss);
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
  TO* yp = y + t * y_stride + c0;
  gain += c0;
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    if constexpr (VEC) {
      const float4 x = reinterpret_cast<const float4*>(xs)[i], g = reinterpret_cast<const float4*>(gain)[i];
      const float4 v = make_float4(x.x * inv * g.x, x.y * inv * g.y, x.z * inv * g.z, x.w * inv * g.w);
      if constexpr (sizeof(TO) == 4) {
        reinterpret_cast<float4*>(yp)[i] = v;
      } else {
        __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        reinterpret_cast<uint2*>(yp)[i] = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
      }
    } else {
      yp[i] = from_f32<TO>(xs[i] * inv * gain[i]);
    }
  }
}

// o, gate: float [T][groups*width] (row strides free); gain: float [groups*width]; y: [T][groups*width] of y_dtype
SGLC_API int sglc_gate_then_norm(const float* o, long long o_stride, const float* gate, long long gate_stride,
                                 const float* gain, void* y, long long y_stride, int y_dtype, int T, int groups,
                                 int width, float eps, int act, cudaStream_t stream) {
  if (T <= 0) return SGLC_OK;
  if (groups <= 0 || width <= 0 || !gate || (act != GN_SILU && act != GN_SIGMOID)) return SGLC_ERR_ARGUMENT;
  if (y_dtype != SGLC_F32 && y_dtype != SGLC_BF16) return SGLC_ERR_ARGUMENT;
  const size_t smem = (size_t)width * sizeof(float);
  if (smem > 200 * 1024 || (long long)T * groups > 0x7fffffffLL) return SGLC_ERR_UNSUPPORTED;
  auto al = [](const void* q, uintptr_t n) { return (reinterpret_cast<uintptr_t>(q) & (n - 1)) == 0; };
  const bool vec = width % 4 == 0 && (o_stride | gate_stride | y_stride) % 4 == 0 && al(o, 16) && al(gate, 16) &&
                   al(gain, 16) && al(y, y_dtype == SGLC_F32 ? 16 : 8);
  const int work = vec ? width / 4 : width;
  int threads = (work + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  const dim3 grid((unsigned)((long long)T * groups));
#define GO(TO, VEC)                                                                                              \
  do {                                                                                                           \
    if (smem > 48 * 1024)                                                                                        \
      cudaFuncSetAttribute(gate_then_norm_kernel<TO, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    return sglc_launch(gate_then_norm_kernel<TO, VEC>, grid, dim3(threads), smem, stream, 1, true, o, o_stride, gate, \
                       gate_stride, gain, (TO*)y, y_stride, groups, width, eps, act);                            \
  } while (0)
  if (y_dtype == SGLC_BF16) {
    if (vec) GO(__nv_bfloat16, true);
    GO(__nv_bfloat16, false);
  }
  if (vec) GO(float, true);
  GO(float, false);
#undef GO
}

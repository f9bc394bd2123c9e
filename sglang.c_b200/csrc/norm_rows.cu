// Row norms in their general form, for the places the LayerNorm-with-bias kernel does not cover:
//   layer form   y = (x - mean) / sqrt(mean((x - mean)^2) + eps) * g (+ b)
//   RMS form     y = x / sqrt(mean(x^2) + eps) * g (+ b)
// gain and bias may each be absent.  The source is float or bfloat16 with a free row stride (a
// column range of a wider buffer: a latent beside the queries of one projection) and an optional
// row gather; statistics are two-pass in 32-bit.  Three destinations:
//   rows      dst[r, :] = y                      (float or bfloat16, free row stride)
//   scatter   dst[dst_rows[r], :] = y            (the rows of a paged cache, by slot)
//   add       dst[r, :] += y                     (float: a norm behind a sublayer, summed into the
//                                                 32-bit residual stream)
// In groups: a row is split into `groups` equal consecutive parts, each normalised by its own
// statistics; gain and bias span the whole row.  A block then takes one part of one row.
// One block a row; the order of a row's additions depends on the row's width only, so a row's
// bits do not depend on what else is in the step.
#include "common.cuh"

SGLC_DEFINE_ERROR_STRING()

enum { NORM_LAYER = 0, NORM_RMS = 1, NORM_COPY = 2 };   // NORM_COPY: the tail's second stage only, no norm

// Four floats at a time (VEC: a 32-bit source whose rows, gains and destination can be read and
// written 16 bytes at a time).  A thread's order of additions differs between the two forms; which
// form runs depends on the row width and the alignment of the buffers, never on the step.
__device__ __forceinline__ float sum4(const float4& v) { return (v.x + v.y) + (v.z + v.w); }
__device__ __forceinline__ float sq4(const float4& v, float mean, float q) {
  float d = v.x - mean; q = fmaf(d, d, q);
  d = v.y - mean; q = fmaf(d, d, q);
  d = v.z - mean; q = fmaf(d, d, q);
  d = v.w - mean; q = fmaf(d, d, q);
  return q;
}
__device__ __forceinline__ float4 norm4(const float4& v, float mean, float inv, const float* gain, const float* bias, int i) {
  float4 y = make_float4(__fmul_rn(v.x - mean, inv), __fmul_rn(v.y - mean, inv), __fmul_rn(v.z - mean, inv),
                         __fmul_rn(v.w - mean, inv));
  if (gain) {
    const float4 g = reinterpret_cast<const float4*>(gain)[i];
    y = make_float4(__fmul_rn(y.x, g.x), __fmul_rn(y.y, g.y), __fmul_rn(y.z, g.z), __fmul_rn(y.w, g.w));
  }
  if (bias) {
    const float4 b = reinterpret_cast<const float4*>(bias)[i];
    y = make_float4(__fadd_rn(y.x, b.x), __fadd_rn(y.y, b.y), __fadd_rn(y.z, b.z), __fadd_rn(y.w, b.w));
  }
  return y;
}
template <typename TO>
__device__ __forceinline__ void store4(TO* p, const float4& y) {
  if constexpr (sizeof(TO) == 4) {
    *reinterpret_cast<float4*>(p) = y;
  } else {
    __nv_bfloat162 h0 = __floats2bfloat162_rn(y.x, y.y), h1 = __floats2bfloat162_rn(y.z, y.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&h0), *reinterpret_cast<uint32_t*>(&h1));
  }
}

template <typename TI, typename TO, bool ADD, bool VEC>
__global__ void norm_rows_kernel(const TI* __restrict__ src, long long src_stride,
                                 const int* __restrict__ src_rows, const float* __restrict__ gain, const float* __restrict__ bias,
                                 TO* __restrict__ dst, long long dst_stride, const int* __restrict__ dst_rows,
                                 int n_rows, int E, float eps, int form, long long dst_row_limit,
                                 int* __restrict__ err, int groups) {
  extern __shared__ __align__(16) float srow[];   // E floats
  __shared__ float red[33];
  // (groups > 1: a block takes one of a row's equal consecutive parts, E being the part's width)
  const int r = blockIdx.x / groups, part = (blockIdx.x % groups) * E;
  if (r >= n_rows) return;
  if (gain) gain += part;
  if (bias) bias += part;
  pdl_launch_dependents();
  pdl_wait();
  const TI* xr = src + (size_t)(src_rows ? src_rows[r] : r) * src_stride + part;
  float s = 0.0f;
  if constexpr (VEC) {
    for (int i = threadIdx.x; i < E / 4; i += blockDim.x) {
      const float4 v = reinterpret_cast<const float4*>(xr)[i];
      reinterpret_cast<float4*>(srow)[i] = v;
      s += sum4(v);
    }
  } else {
    for (int i = threadIdx.x; i < E; i += blockDim.x) {
      const float v = to_f32(xr[i]);
      srow[i] = v;
      s += v;
    }
  }
  float mean = 0.0f;
  if (form == NORM_LAYER) mean = block_sum(s, red) / (float)E;
  else __syncthreads();
  float q = 0.0f;
  if constexpr (VEC) {
    for (int i = threadIdx.x; i < E / 4; i += blockDim.x) q = sq4(reinterpret_cast<const float4*>(srow)[i], mean, q);
  } else {
    for (int i = threadIdx.x; i < E; i += blockDim.x) {
      const float d = srow[i] - mean;
      q = fmaf(d, d, q);
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(q, red) / (float)E + eps);
  long long row = r;
  if (dst_rows) {
    row = dst_rows[r];
    if (row < 0 || !sglc_index_ok(row, dst_row_limit, err)) return;
  }
  TO* o = dst + (size_t)row * dst_stride + part;
  if constexpr (VEC) {
    for (int i = threadIdx.x; i < E / 4; i += blockDim.x) {
      float4 y = norm4(reinterpret_cast<const float4*>(srow)[i], mean, inv, gain, bias, i);
      if constexpr (ADD) {
        const float4 x = reinterpret_cast<const float4*>(o)[i];
        y = make_float4(__fadd_rn(x.x, y.x), __fadd_rn(x.y, y.y), __fadd_rn(x.z, y.z), __fadd_rn(x.w, y.w));
      }
      store4<TO>(o + 4 * i, y);
    }
  } else {
    for (int i = threadIdx.x; i < E; i += blockDim.x) {
      // (explicit roundings: the fused tail below must give the same bits, whatever either compiles to)
      float y = __fmul_rn(srow[i] - mean, inv);
      if (gain) y = __fmul_rn(y, gain[i]);
      if (bias) y = __fadd_rn(y, bias[i]);
      if (ADD) o[i] = from_f32<TO>(__fadd_rn(to_f32(o[i]), y));
      else o[i] = from_f32<TO>(y);
    }
  }
}

// The tail of a sublayer in one launch, a block a row:
//   x += norm_post(y) * g_post                                   (x: the 32-bit stream)
//   [mix]   hist[n_terms-1] = x;  x = sum_j w[j] * hist[j]        (a depth-weighted average, j ascending)
//   [next]  h = norm_next(x) * g_next                            (the norm ahead of the next sublayer;
//                                                                  form NORM_COPY: h = x in h's precision)
// The same arithmetic in the same order as the three kernels it stands for, so the bits are theirs.
template <typename TO, bool VEC>
__global__ void norm_add_tail_kernel(const float* __restrict__ y, long long y_stride,
                                     const float* __restrict__ g_post, float eps_post, int form_post,
                                     float* __restrict__ x, float* __restrict__ hist, long long hist_block,
                                     int n_terms, const float* __restrict__ mix_w,
                                     const float* __restrict__ g_next, float eps_next, int form_next,
                                     TO* __restrict__ h, long long h_stride, int n_rows, int E) {
  extern __shared__ __align__(16) float srow[];   // E floats
  __shared__ float red[33];
  const int r = blockIdx.x;
  if (r >= n_rows) return;
  pdl_launch_dependents();
  pdl_wait();
  const float* yr = y + (size_t)r * y_stride;
  const int n_it = VEC ? E / 4 : E;
  float s = 0.0f;
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    if constexpr (VEC) {
      const float4 v = reinterpret_cast<const float4*>(yr)[i];
      reinterpret_cast<float4*>(srow)[i] = v;
      s += sum4(v);
    } else {
      const float v = yr[i];
      srow[i] = v;
      s += v;
    }
  }
  float mean = 0.0f;
  if (form_post == NORM_LAYER) mean = block_sum(s, red) / (float)E;
  else __syncthreads();
  float q = 0.0f;
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    if constexpr (VEC) {
      q = sq4(reinterpret_cast<const float4*>(srow)[i], mean, q);
    } else {
      const float d = srow[i] - mean;
      q = fmaf(d, d, q);
    }
  }
  float inv = 1.0f / sqrtf(block_sum(q, red) / (float)E + eps_post);
  float* xr = x + (size_t)r * E;
  s = 0.0f;
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    if constexpr (VEC) {
      float4 v = norm4(reinterpret_cast<const float4*>(srow)[i], mean, inv, g_post, nullptr, i);
      const float4 x0 = reinterpret_cast<const float4*>(xr)[i];
      v = make_float4(__fadd_rn(x0.x, v.x), __fadd_rn(x0.y, v.y), __fadd_rn(x0.z, v.z), __fadd_rn(x0.w, v.w));
      if (n_terms > 0) {
        const size_t at = ((size_t)r * E) / 4 + i;
        reinterpret_cast<float4*>(hist + (size_t)(n_terms - 1) * hist_block)[at] = v;
        if (n_terms > 1) {
          float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
          for (int j = 0; j < n_terms - 1; j++) {
            const float4 hv = reinterpret_cast<const float4*>(hist + (size_t)j * hist_block)[at];
            const float wj = mix_w[j];
            acc.x = fmaf(wj, hv.x, acc.x); acc.y = fmaf(wj, hv.y, acc.y);
            acc.z = fmaf(wj, hv.z, acc.z); acc.w = fmaf(wj, hv.w, acc.w);
          }
          const float wl = mix_w[n_terms - 1];
          v = make_float4(fmaf(wl, v.x, acc.x), fmaf(wl, v.y, acc.y), fmaf(wl, v.z, acc.z), fmaf(wl, v.w, acc.w));
        }
      }
      reinterpret_cast<float4*>(xr)[i] = v;
      reinterpret_cast<float4*>(srow)[i] = v;
      s += sum4(v);
    } else {
      float v = __fmul_rn(srow[i] - mean, inv);
      if (g_post) v = __fmul_rn(v, g_post[i]);
      v = __fadd_rn(xr[i], v);
      if (n_terms > 0) {
        const size_t at = (size_t)r * E + i;
        hist[(size_t)(n_terms - 1) * hist_block + at] = v;
        if (n_terms > 1) {
          float acc = 0.0f;
          for (int j = 0; j < n_terms - 1; j++) acc = fmaf(mix_w[j], hist[(size_t)j * hist_block + at], acc);
          v = fmaf(mix_w[n_terms - 1], v, acc);
        }
      }
      xr[i] = v;
      srow[i] = v;
      s += v;
    }
  }
  if (!h) return;
  if (form_next == NORM_COPY) {
    __syncthreads();
    TO* hc = h + (size_t)r * h_stride;
    for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
      if constexpr (VEC) store4<TO>(hc + 4 * i, reinterpret_cast<const float4*>(srow)[i]);
      else hc[i] = from_f32<TO>(srow[i]);
    }
    return;
  }
  mean = 0.0f;
  if (form_next == NORM_LAYER) mean = block_sum(s, red) / (float)E;
  else __syncthreads();
  q = 0.0f;
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    if constexpr (VEC) {
      q = sq4(reinterpret_cast<const float4*>(srow)[i], mean, q);
    } else {
      const float d = srow[i] - mean;
      q = fmaf(d, d, q);
    }
  }
  inv = 1.0f / sqrtf(block_sum(q, red) / (float)E + eps_next);
  TO* hr = h + (size_t)r * h_stride;
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    if constexpr (VEC) {
      store4<TO>(hr + 4 * i, norm4(reinterpret_cast<const float4*>(srow)[i], mean, inv, g_next, nullptr, i));
    } else {
      float v = __fmul_rn(srow[i] - mean, inv);
      if (g_next) v = __fmul_rn(v, g_next[i]);
      hr[i] = from_f32<TO>(v);
    }
  }
}

// y: float [n_rows][y_stride]; x: float [n_rows][E] contiguous; hist (n_terms > 0): float blocks of
// hist_block elements, block j holding [n_rows][E]; h (may be null): [n_rows][h_stride] of h_dtype.
static inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

SGLC_API int sglc_norm_add_tail(const float* y, long long y_stride, const float* g_post, float eps_post,
                                int form_post, float* x, float* hist, long long hist_block, int n_terms,
                                const float* mix_w, const float* g_next, float eps_next, int form_next, void* h,
                                long long h_stride, int h_dtype, int n_rows, int E, cudaStream_t stream) {
  if (n_rows <= 0) return SGLC_OK;
  if (E <= 0 || n_terms < 0 || (n_terms > 0 && !hist) || (n_terms > 1 && !mix_w)) return SGLC_ERR_ARGUMENT;
  if (h && h_dtype != SGLC_F32 && h_dtype != SGLC_BF16) return SGLC_ERR_ARGUMENT;
  const size_t smem = (size_t)E * sizeof(float);
  if (smem > 200 * 1024) return SGLC_ERR_UNSUPPORTED;
  const int threads = E >= 2048 ? 512 : (E >= 512 ? 256 : (E >= 128 ? 128 : (E >= 64 ? 64 : 32)));
  const bool vec = E % 4 == 0 && y_stride % 4 == 0 && al16(y) && al16(x) && al16(g_post) && al16(g_next) &&
                   (!hist || (al16(hist) && hist_block % 4 == 0)) &&
                   (!h || (h_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(h) & (h_dtype == SGLC_F32 ? 15 : 7)) == 0));
#define TAIL(TO, VEC)                                                                                          \
  do {                                                                                                         \
    if (smem > 48 * 1024)                                                                                      \
      cudaFuncSetAttribute(norm_add_tail_kernel<TO, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    return sglc_launch(norm_add_tail_kernel<TO, VEC>, dim3(n_rows), dim3(threads), smem, stream, 1, true, y,    \
                       y_stride, g_post, eps_post, form_post, x, hist, hist_block, n_terms, mix_w, g_next,      \
                       eps_next, form_next, (TO*)h, h_stride, n_rows, E);                                       \
  } while (0)
  if (h && h_dtype == SGLC_BF16) {
    if (vec) TAIL(__nv_bfloat16, true);
    TAIL(__nv_bfloat16, false);
  }
  if (vec) TAIL(float, true);
  TAIL(float, false);
#undef TAIL
}

// form: 0 layer, 1 RMS.  src_rows: null, or the source row of every output row (a gather).  src_dtype/dst_dtype: SGLC_F32 or SGLC_BF16.  dst_rows: null, or the
// destination row of every source row (negative: the row is skipped); dst_row_limit: rows the
// destination holds (the bounds-check build compares).  add != 0: dst (float) += y.
SGLC_API int sglc_norm_rows_grouped(const void* src, long long src_stride, int src_dtype, const int* src_rows,
                                    const float* gain,
                                    const float* bias, void* dst, long long dst_stride, int dst_dtype,
                                    const int* dst_rows, long long dst_row_limit, int n_rows, int E_row, float eps,
                                    int form, int add, int groups, int* err, cudaStream_t stream) {
  if (n_rows <= 0) return SGLC_OK;
  if (E_row <= 0 || groups <= 0 || E_row % groups != 0 || (form != NORM_LAYER && form != NORM_RMS)) return SGLC_ERR_ARGUMENT;
  if ((long long)n_rows * groups > 0x7fffffffLL) return SGLC_ERR_UNSUPPORTED;
  const int E = E_row / groups;            // what a block normalises
  if (add && dst_dtype != SGLC_F32) return SGLC_ERR_ARGUMENT;
  const size_t smem = (size_t)E * sizeof(float);
  if (smem > 200 * 1024) return SGLC_ERR_UNSUPPORTED;
  const bool vec = src_dtype == SGLC_F32 && E % 4 == 0 && src_stride % 4 == 0 && dst_stride % 4 == 0 && al16(src) &&
                   al16(gain) && al16(bias) &&
                   (reinterpret_cast<uintptr_t>(dst) & (dst_dtype == SGLC_F32 ? 15 : 7)) == 0;
  // (a narrow part read four floats a thread fills no second warp: one warp then, whose sums are the
  // same bits, since the second warp only added zeros)
  const int threads = E >= 2048 ? 512 : (E >= 512 ? 256 : (E >= 128 ? 128 : (E >= 64 && !vec ? 64 : 32)));
#define LAUNCH(TI, TO, ADD) \
  do {                      \
    if (vec) LAUNCH_V(float, TO, ADD, true); \
    LAUNCH_V(TI, TO, ADD, false);            \
  } while (0)
#define LAUNCH_V(TI, TO, ADD, VEC)                                                                   \
  do {                                                                                               \
    if (smem > 48 * 1024)                                                                            \
      cudaFuncSetAttribute(norm_rows_kernel<TI, TO, ADD, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                           (int)smem);                                                               \
    return sglc_launch(norm_rows_kernel<TI, TO, ADD, VEC>, dim3(n_rows * groups), dim3(threads), smem, stream, 1, \
                       true, (const TI*)src, src_stride, src_rows, gain, bias, (TO*)dst, dst_stride, dst_rows,  \
                       n_rows, E, eps, form, dst_row_limit, err, groups);                             \
  } while (0)
  if (src_dtype == SGLC_F32) {
    if (add) LAUNCH(float, float, true);
    if (dst_dtype == SGLC_F32) LAUNCH(float, float, false);
    if (dst_dtype == SGLC_BF16) LAUNCH(float, __nv_bfloat16, false);
  } else if (src_dtype == SGLC_BF16) {
    if (add) LAUNCH(__nv_bfloat16, float, true);
    if (dst_dtype == SGLC_F32) LAUNCH(__nv_bfloat16, float, false);
    if (dst_dtype == SGLC_BF16) LAUNCH(__nv_bfloat16, __nv_bfloat16, false);
  }
#undef LAUNCH
#undef LAUNCH_V
  return SGLC_ERR_ARGUMENT;
}

SGLC_API int sglc_norm_rows(const void* src, long long src_stride, int src_dtype, const int* src_rows,
                            const float* gain,
                            const float* bias, void* dst, long long dst_stride, int dst_dtype,
                            const int* dst_rows, long long dst_row_limit, int n_rows, int E, float eps,
                            int form, int add, int* err, cudaStream_t stream) {
  return sglc_norm_rows_grouped(src, src_stride, src_dtype, src_rows, gain, bias, dst, dst_stride, dst_dtype, dst_rows,
                                dst_row_limit, n_rows, E, eps, form, add, 1, err, stream);
}

// Two RMS norms of the same rows (parallel sublayers with a norm each) and, on the first one's
// result, a token shift, in one launch, a block a token:
//   h_t = x_t / sqrt(mean(x_t^2) + eps) * g1;   y1_t = h_t + (h_(t-1) - h_t) * mu;   y2_t likewise with g2
// h_(t-1) is the token before of the same request, before its own shift; zero ahead of the first
// token, and `prev[slot]` (kept in 32-bit) ahead of a portion's first.  The block of a portion's
// FIRST token is the only one that touches the slot: it reads what the portion before left and then
// writes the h of the portion's last token, which it norms itself, so nothing waits for another block.
// Without mu: y1 = h.  Without y2: one norm.
template <typename TO, bool VEC>
__global__ void norm_pair_shift_kernel(const float* __restrict__ x, const float* __restrict__ g1,
                                       const float* __restrict__ g2, const float* __restrict__ mu, float eps,
                                       float* __restrict__ prev, const int* __restrict__ token_req,
                                       const int* __restrict__ q_start, const int* __restrict__ state_slots,
                                       TO* __restrict__ y1, long long y1_stride, TO* __restrict__ y2,
                                       long long y2_stride, int E, int n_slots, int* __restrict__ err) {
  extern __shared__ __align__(16) float srow[];   // the token's row; with mu, then the other row
  __shared__ float red[2][33];
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  pdl_launch_dependents();
  // (the step's own arrays: no kernel of the step writes them)
  int first = 0, last = 0, slot = -1;
  if (mu) {
    const int r = token_req[t];
    first = q_start[r];
    last = q_start[r + 1] - 1;
    slot = state_slots[r];
  }
  const bool head = mu && t == first;             // this block serves the slot
  const int other = !mu ? -1 : head ? last : t - 1;
  float* orow = srow + E;
  const int n_it = VEC ? E / 4 : E;
  pdl_wait();
  const float* xr = x + (size_t)t * E;
  const float* xo = x + (size_t)(other < 0 ? t : other) * E;
  const bool two = mu && other != t;              // (a single token's own row serves as the last one)
  float qa = 0.0f, qb = 0.0f;
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    if constexpr (VEC) {
      const float4 v = reinterpret_cast<const float4*>(xr)[i];
      reinterpret_cast<float4*>(srow)[i] = v;
      qa = sq4(v, 0.0f, qa);
      if (two) {
        const float4 o = reinterpret_cast<const float4*>(xo)[i];
        reinterpret_cast<float4*>(orow)[i] = o;
        qb = sq4(o, 0.0f, qb);
      }
    } else {
      const float v = xr[i];
      srow[i] = v;
      qa = fmaf(v, v, qa);
      if (two) {
        const float o = xo[i];
        orow[i] = o;
        qb = fmaf(o, o, qb);
      }
    }
  }
  // both sums at once; the order of additions depends on the width only
  qa = warp_sum(qa);
  qb = warp_sum(qb);
  if (lane == 0) { red[0][warp] = qa; red[1][warp] = qb; }
  __syncthreads();
  qa = 0.0f; qb = 0.0f;
  for (int w = 0; w < nw; w++) { qa += red[0][w]; qb += red[1][w]; }
  const float ia = 1.0f / sqrtf(qa / (float)E + eps);
  const float ib = two ? 1.0f / sqrtf(qb / (float)E + eps) : ia;
  const float* brow = two ? orow : srow;
  float* ps = nullptr;
  if (head) {
    if (!sglc_index_ok(slot, n_slots, err)) return;
    ps = prev + (size_t)slot * E;
  }
  TO* o1 = y1 + (size_t)t * y1_stride;
  TO* o2 = y2 ? y2 + (size_t)t * y2_stride : nullptr;
  // (a thread reads and writes the same columns of the rows it staged, so nothing more is waited for)
  for (int i = threadIdx.x; i < n_it; i += blockDim.x) {
    if constexpr (VEC) {
      const float4 v = reinterpret_cast<const float4*>(srow)[i];
      float4 h = norm4(v, 0.0f, ia, g1, nullptr, i);
      if (mu) {
        const float4 hb = norm4(reinterpret_cast<const float4*>(brow)[i], 0.0f, ib, g1, nullptr, i);
        float4 p = hb;
        if (head) {
          p = reinterpret_cast<float4*>(ps)[i];
          reinterpret_cast<float4*>(ps)[i] = hb;
        }
        const float4 m = reinterpret_cast<const float4*>(mu)[i];
        h = make_float4(fmaf(p.x - h.x, m.x, h.x), fmaf(p.y - h.y, m.y, h.y), fmaf(p.z - h.z, m.z, h.z),
                        fmaf(p.w - h.w, m.w, h.w));
      }
      store4<TO>(o1 + 4 * i, h);
      if (o2) store4<TO>(o2 + 4 * i, norm4(v, 0.0f, ia, g2, nullptr, i));
    } else {
      const float n = __fmul_rn(srow[i], ia);
      float h = g1 ? __fmul_rn(n, g1[i]) : n;
      if (mu) {
        float hb = __fmul_rn(brow[i], ib);
        if (g1) hb = __fmul_rn(hb, g1[i]);
        float p = hb;
        if (head) {
          p = ps[i];
          ps[i] = hb;
        }
        h = fmaf(p - h, mu[i], h);
      }
      o1[i] = from_f32<TO>(h);
      if (o2) o2[i] = from_f32<TO>(g2 ? __fmul_rn(n, g2[i]) : n);
    }
  }
}

// The same for steps of many tokens (four floats at a time): a block takes PAIR_TOKENS consecutive
// tokens, a warp each, and one warp more for the token ahead of them, so a row is read once by a block
// that needs it twice.  A portion's first token finds its slot and its portion's last row by itself.
constexpr int PAIR_TOKENS = 8;

template <typename TO>
__global__ void __launch_bounds__((PAIR_TOKENS + 1) * 32)
norm_pair_shift_rows_kernel(const float* __restrict__ x, const float* __restrict__ g1, const float* __restrict__ g2,
                            const float* __restrict__ mu, float eps, float* __restrict__ prev,
                            const int* __restrict__ token_req, const int* __restrict__ q_start,
                            const int* __restrict__ state_slots, TO* __restrict__ y1, long long y1_stride,
                            TO* __restrict__ y2, long long y2_stride, int T, int E, int n_slots, int* __restrict__ err) {
  extern __shared__ __align__(16) float rows[];   // [PAIR_TOKENS + 1][E]
  __shared__ float inv_s[PAIR_TOKENS + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * PAIR_TOKENS + warp - 1;      // (warp 0: the token ahead of the block's)
  pdl_launch_dependents();
  bool head = false;
  int last = t, slot = -1;
  if (mu && warp > 0 && t < T) {
    const int r = token_req[t];
    head = t == q_start[r];
    last = q_start[r + 1] - 1;
    slot = state_slots[r];
  }
  pdl_wait();
  const int n_it = E / 4;
  float4* mine = reinterpret_cast<float4*>(rows + (size_t)warp * E);
  if (t >= 0 && t < T && (warp > 0 || mu)) {
    float q = 0.0f;
    for (int i = lane; i < n_it; i += 32) {
      const float4 v = reinterpret_cast<const float4*>(x + (size_t)t * E)[i];
      mine[i] = v;
      q = sq4(v, 0.0f, q);
    }
    q = warp_sum(q);
    if (lane == 0) inv_s[warp] = 1.0f / sqrtf(q / (float)E + eps);
  }
  __syncthreads();
  if (warp == 0 || t >= T) return;
  const float ia = inv_s[warp];
  float ib = warp > 0 ? inv_s[warp - 1] : 0.0f;
  const float4* before = reinterpret_cast<const float4*>(rows + (size_t)(warp - 1) * E);
  float4* ps = nullptr;
  if (head) {
    if (!sglc_index_ok(slot, n_slots, err)) return;
    ps = reinterpret_cast<float4*>(prev + (size_t)slot * E);
    before = reinterpret_cast<const float4*>(x + (size_t)last * E);      // what the slot takes
    float q = 0.0f;
    for (int i = lane; i < n_it; i += 32) q = sq4(before[i], 0.0f, q);
    ib = 1.0f / sqrtf(warp_sum(q) / (float)E + eps);
  }
  TO* o1 = y1 + (size_t)t * y1_stride;
  TO* o2 = y2 ? y2 + (size_t)t * y2_stride : nullptr;
  for (int i = lane; i < n_it; i += 32) {
    const float4 v = mine[i];
    float4 h = norm4(v, 0.0f, ia, g1, nullptr, i);
    if (mu) {
      const float4 hb = norm4(before[i], 0.0f, ib, g1, nullptr, i);
      float4 p = hb;
      if (head) {
        p = ps[i];
        ps[i] = hb;
      }
      const float4 m = reinterpret_cast<const float4*>(mu)[i];
      h = make_float4(fmaf(p.x - h.x, m.x, h.x), fmaf(p.y - h.y, m.y, h.y), fmaf(p.z - h.z, m.z, h.z),
                      fmaf(p.w - h.w, m.w, h.w));
    }
    store4<TO>(o1 + 4 * i, h);
    if (o2) store4<TO>(o2 + 4 * i, norm4(v, 0.0f, ia, g2, nullptr, i));
  }
}
constexpr int PAIR_ROWS_MIN = 296;      // tokens from which the form above is used: two blocks' worth of rows an SM

// x: float [T][E] contiguous; g1, g2, mu: float [E] (g2 with y2 only; mu may be null); prev: float
// [n_slots][E] (with mu); y1, y2 (y2 may be null): [T][stride] of out_dtype.
SGLC_API int sglc_norm_pair_shift(const float* x, const float* g1, const float* g2, const float* mu, float eps,
                                  float* prev, const int* token_req, const int* q_start, const int* state_slots,
                                  void* y1, long long y1_stride, void* y2, long long y2_stride, int out_dtype, int T,
                                  int E, int n_slots, int* err, cudaStream_t stream) {
  if (T <= 0) return SGLC_OK;
  if (E <= 0 || !y1 || (mu && (!prev || !token_req || !q_start || !state_slots))) return SGLC_ERR_ARGUMENT;
  if (out_dtype != SGLC_F32 && out_dtype != SGLC_BF16) return SGLC_ERR_ARGUMENT;
  const size_t smem = (size_t)E * (mu ? 2 : 1) * sizeof(float);
  if (smem > 200 * 1024) return SGLC_ERR_UNSUPPORTED;
  const int threads = E >= 2048 ? 512 : (E >= 512 ? 256 : (E >= 128 ? 128 : (E >= 64 ? 64 : 32)));
  const int oa = out_dtype == SGLC_F32 ? 15 : 7;
  const bool vec = E % 4 == 0 && al16(x) && al16(g1) && al16(g2) && al16(mu) && al16(prev) && y1_stride % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(y1) & oa) == 0 &&
                   (!y2 || (y2_stride % 4 == 0 && (reinterpret_cast<uintptr_t>(y2) & oa) == 0));
  const size_t smem_rows = (size_t)(PAIR_TOKENS + 1) * E * sizeof(float);
  if (vec && T >= PAIR_ROWS_MIN && smem_rows <= 100 * 1024) {
    const dim3 grid((T + PAIR_TOKENS - 1) / PAIR_TOKENS), block((PAIR_TOKENS + 1) * 32);
#define ROWS(TO)                                                                                                  \
  do {                                                                                                            \
    if (smem_rows > 48 * 1024)                                                                                    \
      cudaFuncSetAttribute(norm_pair_shift_rows_kernel<TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_rows); \
    return sglc_launch(norm_pair_shift_rows_kernel<TO>, grid, block, smem_rows, stream, 1, true, x, g1, g2, mu, eps, prev, \
                       token_req, q_start, state_slots, (TO*)y1, y1_stride, (TO*)y2, y2_stride, T, E, n_slots, err); \
  } while (0)
    if (out_dtype == SGLC_BF16) ROWS(__nv_bfloat16);
    ROWS(float);
#undef ROWS
  }
#define PAIR(TO, VEC)                                                                                            \
  do {                                                                                                           \
    if (smem > 48 * 1024)                                                                                        \
      cudaFuncSetAttribute(norm_pair_shift_kernel<TO, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    return sglc_launch(norm_pair_shift_kernel<TO, VEC>, dim3(T), dim3(threads), smem, stream, 1, true, x, g1, g2, mu, \
                       eps, prev, token_req, q_start, state_slots, (TO*)y1, y1_stride, (TO*)y2, y2_stride, E, n_slots, \
                       err);                                                                                     \
  } while (0)
  if (out_dtype == SGLC_BF16) {
    if (vec) PAIR(__nv_bfloat16, true);
    PAIR(__nv_bfloat16, false);
  }
  if (vec) PAIR(float, true);
  PAIR(float, false);
#undef PAIR
}

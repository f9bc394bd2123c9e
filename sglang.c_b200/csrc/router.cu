// Routing of a mixture of experts for the tokens of a step, from 32-bit router logits z [T][E]:
//   s = sigmoid(z);   choice = s + correction          (the correction only steers the choice)
//   experts form `n_groups` equal groups of neighbours; a group's score is the sum of its two
//   largest choice scores; only experts of the `keep` best groups can be chosen (the others
//   count as minus infinity); the `top` largest choice scores among them are chosen;
//   a chosen expert's weight is its s (times `weight_scale`; with `renorm` the chosen weights
//   are first divided by their sum plus `renorm_eps`).
// `score_fn` 1: s = softmax(z) over all experts instead of the sigmoid.
// `group_fn` 1: a group's score is its largest choice score instead of the sum of its two largest.
// Of the E experts the last `n_pass` may be ones that hand their input on as it is: `pass` [T] (if
// given) takes the sum of the token's weights for them.
// Ties go to the lower index.  Results: dense [T][E] weights (zero where not chosen), and the
// chosen ids and weights [T][top] in order of choice.  A warp a token, a lane every 32nd expert; all
// 32-bit.  The logits either come from a product of the caller's, or are made here from the token's
// row and the router's matrix (a block a token: its warps take the experts' dot products in turn, then
// one of them routes), where re-reading a small matrix costs less than a launch of its own.
#include "common.cuh"

SGLC_DEFINE_ERROR_STRING()

constexpr int ROUTER_MAX_EXPERTS = 256;
constexpr int ROUTER_MAX_GROUPS = 64;
constexpr int ROUTER_PER_LANE = ROUTER_MAX_EXPERTS / 32;
constexpr int ROUTER_TOKENS = 4;      // tokens of a block where the logits are given
constexpr int ROUTER_WARPS = 8;       // warps of a token where they are not

struct RouterArgs {
  const float* z; long long z_stride;        // given logits, or null
  const void* h; long long h_stride;         // rows [T][K] and matrix [E][K] to make them from
  const void* w; int K;
  const float* correction;
  float* dense; long long dense_stride;
  int* ids; float* wts;
  int T, E, top, n_groups, keep, renorm, score_fn, group_fn, n_pass;
  float weight_scale, renorm_eps;
  float* pass;
};

// The largest value of the warp and the lowest index that has it.
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) { v = ov; i = oi; }
  }
}

// One warp routes token t.  zs: its E logits; cs: E floats of scratch (both in shared memory).
__device__ __forceinline__ void route(const RouterArgs& a, int t, const float* zs, float* cs) {
  const int lane = threadIdx.x & 31, E = a.E;
  constexpr int NONE = 1 << 30;
  float s[ROUTER_PER_LANE], c[ROUTER_PER_LANE];
  float zmax = -INFINITY, zden = 0.0f;
  if (a.score_fn == 1) {                       // softmax: the largest logit and the sum of exponentials
#pragma unroll
    for (int i = 0; i < ROUTER_PER_LANE; i++)
      if (lane + 32 * i < E) zmax = fmaxf(zmax, zs[lane + 32 * i]);
    zmax = warp_max(zmax);
#pragma unroll
    for (int i = 0; i < ROUTER_PER_LANE; i++)
      if (lane + 32 * i < E) zden += expf(zs[lane + 32 * i] - zmax);
    zden = warp_sum(zden);
  }
#pragma unroll
  for (int i = 0; i < ROUTER_PER_LANE; i++) {
    const int e = lane + 32 * i;
    s[i] = 0.0f;
    c[i] = -INFINITY;
    if (e < E) {
      s[i] = a.score_fn == 1 ? expf(zs[e] - zmax) / zden : 1.0f / (1.0f + expf(-zs[e]));
      c[i] = s[i] + (a.correction ? a.correction[e] : 0.0f);
    }
  }
  if (a.n_groups > 1 && a.keep < a.n_groups) {
    const int per = E / a.n_groups;
#pragma unroll
    for (int i = 0; i < ROUTER_PER_LANE; i++)
      if (lane + 32 * i < E) cs[lane + 32 * i] = c[i];
    __syncwarp();
    float g[2] = {-INFINITY, -INFINITY};       // a lane scores groups lane and lane + 32
    for (int n = 0; n < 2; n++) {
      const int gi = lane + 32 * n;
      if (gi >= a.n_groups) continue;
      float x = -INFINITY, y = -INFINITY;      // largest, second largest
      for (int e = gi * per; e < (gi + 1) * per; e++) {
        const float v = cs[e];
        if (v > x) { y = x; x = v; }
        else if (v > y) y = v;
      }
      g[n] = per > 1 && a.group_fn == 0 ? x + y : x;
    }
    // the groups that stay: the `keep` best; the others' experts leave the choice
    unsigned long long kept = 0ull;
    bool taken[2] = {lane >= a.n_groups, lane + 32 >= a.n_groups};
    for (int n = 0; n < a.keep; n++) {
      float v = -INFINITY;
      int at = NONE;
      for (int m = 0; m < 2; m++)
        if (!taken[m] && (at == NONE || g[m] > v)) { v = g[m]; at = lane + 32 * m; }
      warp_argmax(v, at);
      if (at == lane) taken[0] = true;
      if (at == lane + 32) taken[1] = true;
      if (at < a.n_groups) kept |= 1ull << at;
    }
#pragma unroll
    for (int i = 0; i < ROUTER_PER_LANE; i++) {
      const int e = lane + 32 * i;
      if (e < E && !((kept >> (e / per)) & 1ull)) c[i] = -INFINITY;
    }
  }
  unsigned chosen = 0u;                        // bit i: expert lane + 32 i is taken
  float sum = 0.0f;
  for (int n = 0; n < a.top; n++) {
    float v = -INFINITY;
    int at = NONE;
#pragma unroll
    for (int i = 0; i < ROUTER_PER_LANE; i++)
      if (lane + 32 * i < E && !((chosen >> i) & 1u) && (at == NONE || c[i] > v)) { v = c[i]; at = lane + 32 * i; }
    warp_argmax(v, at);
    float w = 0.0f;
#pragma unroll
    for (int i = 0; i < ROUTER_PER_LANE; i++)
      if (at == lane + 32 * i) { chosen |= 1u << i; w = s[i]; }
    w = __shfl_sync(0xffffffffu, w, at & 31);
    sum += w;
    if (lane == 0) a.ids[(size_t)t * a.top + n] = at;
    if (lane == (n & 31)) cs[n] = w;           // (in order of choice; scaled below)
  }
  const float f = (a.renorm ? 1.0f / (sum + a.renorm_eps) : 1.0f) * a.weight_scale;
  __syncwarp();
  for (int n = lane; n < a.top; n += 32) a.wts[(size_t)t * a.top + n] = cs[n] * f;
  float handed_on = 0.0f;
#pragma unroll
  for (int i = 0; i < ROUTER_PER_LANE; i++) {
    const int e = lane + 32 * i;
    if (e >= E) continue;
    const float w = (chosen >> i) & 1u ? s[i] * f : 0.0f;
    a.dense[(size_t)t * a.dense_stride + e] = w;
    if (e >= E - a.n_pass) handed_on += w;
  }
  if (a.pass) {
    handed_on = warp_sum(handed_on);
    if (lane == 0) a.pass[t] = handed_on;
  }
}

__global__ void __launch_bounds__(ROUTER_TOKENS * 32)
router_kernel(const RouterArgs a) {
  __shared__ float zs[ROUTER_TOKENS][ROUTER_MAX_EXPERTS], cs[ROUTER_TOKENS][ROUTER_MAX_EXPERTS];
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * ROUTER_TOKENS + warp;
  pdl_wait();
  if (t >= a.T) return;
  for (int e = lane; e < a.E; e += 32) zs[warp][e] = a.z[(size_t)t * a.z_stride + e];
  __syncwarp();
  route(a, t, zs[warp], cs[warp]);
}

__device__ __forceinline__ float dot_part(const float* h, const float* w, int K, int lane) {
  float acc = 0.0f;
  for (int k = lane; k < K; k += 32) acc = fmaf(h[k], w[k], acc);
  return acc;
}
__device__ __forceinline__ float dot_part(const __nv_bfloat16* h, const __nv_bfloat16* w, int K, int lane) {
  float a0 = 0.0f, a1 = 0.0f;
  if (K % 8 == 0 && ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(w)) & 15) == 0) {
    for (int k = lane; k < K / 8; k += 32) {
      const uint4 u = reinterpret_cast<const uint4*>(h)[k], v = reinterpret_cast<const uint4*>(w)[k];
      const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&u);
      const __nv_bfloat162* q = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const float2 x = __bfloat1622float2(p[j]), y = __bfloat1622float2(q[j]);
        a0 = fmaf(x.x, y.x, a0);
        a1 = fmaf(x.y, y.y, a1);
      }
    }
    return a0 + a1;
  }
  for (int k = lane; k < K; k += 32) a0 = fmaf(to_f32(h[k]), to_f32(w[k]), a0);
  return a0;
}

template <typename TA>
__global__ void __launch_bounds__(ROUTER_WARPS * 32)
router_product_kernel(const RouterArgs a) {
  __shared__ float zs[ROUTER_MAX_EXPERTS], cs[ROUTER_MAX_EXPERTS];
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x;
  pdl_wait();
  const TA* h = static_cast<const TA*>(a.h) + (size_t)t * a.h_stride;
  for (int e = warp; e < a.E; e += ROUTER_WARPS) {
    const float z = warp_sum(dot_part(h, static_cast<const TA*>(a.w) + (size_t)e * a.K, a.K, lane));
    if (lane == 0) zs[e] = z;
  }
  __syncthreads();
  if (warp == 0) route(a, t, zs, cs);
}

static int router_check(const RouterArgs& a) {
  if (a.E <= 0 || a.top <= 0 || a.top > a.E || a.n_groups < 1 || a.E % a.n_groups != 0 || a.keep < 1 || a.keep > a.n_groups)
    return SGLC_ERR_ARGUMENT;
  if (a.E > ROUTER_MAX_EXPERTS || a.n_groups > ROUTER_MAX_GROUPS) return SGLC_ERR_UNSUPPORTED;
  if (a.n_groups > 1 && a.keep < a.n_groups && a.top > a.keep * (a.E / a.n_groups)) return SGLC_ERR_ARGUMENT;
  if ((a.score_fn != 0 && a.score_fn != 1) || (a.group_fn != 0 && a.group_fn != 1) || a.n_pass < 0 || a.n_pass > a.E)
    return SGLC_ERR_ARGUMENT;
  return SGLC_OK;
}

SGLC_API int sglc_router_pass(const float* z, long long z_stride, const float* correction, float* dense,
                              long long dense_stride, int* ids, float* wts, int T, int E, int top, int n_groups,
                              int keep, int renorm, float weight_scale, int score_fn, float renorm_eps,
                              int group_fn, int n_pass, float* pass, cudaStream_t stream) {
  if (T <= 0) return SGLC_OK;
  RouterArgs a = {};
  a.z = z; a.z_stride = z_stride; a.correction = correction; a.dense = dense; a.dense_stride = dense_stride;
  a.ids = ids; a.wts = wts; a.T = T; a.E = E; a.top = top; a.n_groups = n_groups; a.keep = keep; a.renorm = renorm;
  a.weight_scale = weight_scale; a.score_fn = score_fn; a.renorm_eps = renorm_eps; a.group_fn = group_fn;
  a.n_pass = n_pass; a.pass = pass;
  const int code = router_check(a);
  if (code != SGLC_OK) return code;
  return sglc_launch(router_kernel, dim3((T + ROUTER_TOKENS - 1) / ROUTER_TOKENS), dim3(ROUTER_TOKENS * 32), 0, stream, 1,
                     true, a);
}

// The same with the logits made here: z = h W^T in 32-bit, h [T][K] (rows h_stride apart) and W [E][K] of
// one dtype.
SGLC_API int sglc_router_product(const void* h, long long h_stride, const void* w, int K, int dtype,
                                 const float* correction, float* dense, long long dense_stride, int* ids, float* wts,
                                 int T, int E, int top, int n_groups, int keep, int renorm, float weight_scale,
                                 int score_fn, float renorm_eps, int group_fn, int n_pass, float* pass,
                                 cudaStream_t stream) {
  if (T <= 0) return SGLC_OK;
  if (!h || !w || K <= 0) return SGLC_ERR_ARGUMENT;
  RouterArgs a = {};
  a.h = h; a.h_stride = h_stride; a.w = w; a.K = K; a.correction = correction; a.dense = dense;
  a.dense_stride = dense_stride; a.ids = ids; a.wts = wts; a.T = T; a.E = E; a.top = top; a.n_groups = n_groups;
  a.keep = keep; a.renorm = renorm; a.weight_scale = weight_scale; a.score_fn = score_fn; a.renorm_eps = renorm_eps;
  a.group_fn = group_fn; a.n_pass = n_pass; a.pass = pass;
  const int code = router_check(a);
  if (code != SGLC_OK) return code;
  if (dtype == SGLC_F32)
    return sglc_launch(router_product_kernel<float>, dim3(T), dim3(ROUTER_WARPS * 32), 0, stream, 1, true, a);
  if (dtype == SGLC_BF16)
    return sglc_launch(router_product_kernel<__nv_bfloat16>, dim3(T), dim3(ROUTER_WARPS * 32), 0, stream, 1, true, a);
  return SGLC_ERR_ARGUMENT;
}

SGLC_API int sglc_router_ext(const float* z, long long z_stride, const float* correction, float* dense,
                             long long dense_stride, int* ids, float* wts, int T, int E, int top, int n_groups,
                             int keep, int renorm, float weight_scale, int score_fn, float renorm_eps,
                             cudaStream_t stream) {
  return sglc_router_pass(z, z_stride, correction, dense, dense_stride, ids, wts, T, E, top, n_groups, keep, renorm,
                          weight_scale, score_fn, renorm_eps, 0, 0, nullptr, stream);
}

SGLC_API int sglc_router(const float* z, long long z_stride, const float* correction, float* dense,
                         long long dense_stride, int* ids, float* wts, int T, int E, int top, int n_groups,
                         int keep, int renorm, float weight_scale, cudaStream_t stream) {
  return sglc_router_ext(z, z_stride, correction, dense, dense_stride, ids, wts, T, E, top, n_groups, keep, renorm,
                         weight_scale, 0, 0.0f, stream);
}

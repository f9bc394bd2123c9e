// The gated matrix-state recurrence with a skip (matrix_state.cu),
//   S <- g_t S + b_t k_t v_t^T,    o_t = S^T q_t + skip v_t,      g_t = exp(-rate b_t), rate = exp(A_log),
// over portions of many tokens, in chunks of SC_Q tokens that do not wait for one another (the state-space
// duality of Mamba-2).  With c_i = sum_{t <= i} log g_t counted from a chunk's start and S_in the state ahead
// of the chunk,
//   o_i = exp(c_i) S_in^T q_i + sum_{j <= i} exp(c_i - c_j) b_j (q_i . k_j) v_j + skip v_i
//   S_out = exp(c_last) S_in + sum_j exp(c_last - c_j) b_j k_j v_j^T
// in three launches: every chunk's own contribution to S_out and its products q_i . k_j (per group, shared by the
// group's heads); a pass over the chunks of each request that turns contributions into states ahead of
// each chunk; the read-outs.  All of it is 32-bit multiply-adds on tiles in shared memory; the sums c_i are kept as
// a pair of floats, so that their differences are as exact as a 32-bit number allows however far c_i has run.
// A token by token walk takes T dependent steps; this takes about as many multiply-adds and no chain.
#include "common.cuh"

SGLC_DEFINE_ERROR_STRING()

constexpr int SC_Q = 64;          // tokens of a chunk
constexpr int SC_V = 64;          // value columns of a tile
constexpr int SC_N = 128;         // state rows of a tile of the contributions
constexpr int SC_LD = SC_Q + 4;   // row stride of tiles that hold a column per token (16-byte rows, lanes on different banks)
constexpr int SC_MAX_DIM = 256;
constexpr int SC_THREADS = 256;

struct ScArgs {
  const float* q; long long q_stride;       // [T][..], group g at columns g*N
  const float* k; long long k_stride;
  const float* v; long long v_stride;       // head h at columns h*V
  const float* b; long long b_stride;       // [T][..], head h at column h: the input weights
  const float* A_log; const float* skip;    // [H]; skip may be null
  float* out; long long out_stride;         // [T][H*V]
  float* state;                             // [n_slots][H][N][V]
  float* S;                                 // [n_chunks][H][N][V]: contributions, then states ahead of the chunks
  float* qk;                                // [n_chunks][G][SC_Q][SC_Q], (i, j)
  float* total;                             // [n_chunks][H]: exp(c_last)
  const int* q_start; const int* state_slots;
  int R, H, G, N, V, n_slots, n_chunks;
  int vec;                                  // rows of q, k, v and out go four entries at a time
  int* err;
};

struct Chunk { int r, t0, len; };

// The step's chunks in order: request after request, each cut from its own first token.  Called by one whole warp.
__device__ __forceinline__ Chunk find_chunk(const ScArgs& p, int c) {
  const int lane = threadIdx.x & 31;
  int before = 0;
  for (int r0 = 0; r0 < p.R; r0 += 32) {
    const int r = r0 + lane;
    int a = 0, n = 0;
    if (r < p.R) {
      a = p.q_start[r];
      n = p.q_start[r + 1] - a;
    }
    const int mine = (n + SC_Q - 1) / SC_Q;
    int incl = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int x = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += x;
    }
    const int lo = before + incl - mine;
    const unsigned hit = __ballot_sync(0xffffffffu, c >= lo && c < lo + mine);
    if (hit) {
      const int src = __ffs(hit) - 1;
      const int ra = __shfl_sync(0xffffffffu, a, src), rn = __shfl_sync(0xffffffffu, n, src), rl = __shfl_sync(0xffffffffu, lo, src);
      const int off = (c - rl) * SC_Q;
      return {r0 + src, ra + off, min(SC_Q, rn - off)};
    }
    before += __shfl_sync(0xffffffffu, incl, 31);
  }
  return {-1, 0, 0};
}

// c_i of a chunk and the input weights, by one whole warp (two neighbouring tokens a lane); tokens behind the
// end: weight zero, no decay.
__device__ __forceinline__ void chunk_sums(const ScArgs& p, int h, const Chunk& ck, float* hi, float* lo, float* bs) {
  const int lane = threadIdx.x & 31;
  const float rate = expf(p.A_log[h]);
  float w[2];
#pragma unroll
  for (int e = 0; e < 2; e++) {
    const int i = 2 * lane + e;
    w[e] = i < ck.len ? p.b[(size_t)(ck.t0 + i) * p.b_stride + h] : 0.0f;
    bs[i] = w[e];
  }
  const double a0 = -(double)(rate * w[0]), a1 = -(double)(rate * w[1]);
  double s = a0 + a1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double x = __shfl_up_sync(0xffffffffu, s, o);
    if (lane >= o) s += x;
  }
  const double c1 = s, c0 = s - a1;
  hi[2 * lane] = (float)c0; lo[2 * lane] = (float)(c0 - (double)(float)c0);
  hi[2 * lane + 1] = (float)c1; lo[2 * lane + 1] = (float)(c1 - (double)(float)c1);
}
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }

// rows i of a chunk, columns 0..n-1 of src, into dst[column][i] (columns up to n_pad and rows behind the chunk: zeros)
__device__ __forceinline__ void stage_columns(const float* src, long long stride, int len, int n, int n_pad, bool vec, float* dst) {
  // (a lane a row: the writes of a warp fall on different banks)
  if (vec) {
    for (int x = threadIdx.x; x < SC_Q * (n_pad / 4); x += SC_THREADS) {
      const int i = x % SC_Q, c = x / SC_Q * 4;
      const float4 v = (i < len && c < n) ? ld4(src + (size_t)i * stride + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      dst[(c + 0) * SC_LD + i] = v.x; dst[(c + 1) * SC_LD + i] = v.y;
      dst[(c + 2) * SC_LD + i] = v.z; dst[(c + 3) * SC_LD + i] = v.w;
    }
  } else {
    for (int x = threadIdx.x; x < SC_Q * n_pad; x += SC_THREADS) {
      const int i = x % SC_Q, c = x / SC_Q;
      dst[c * SC_LD + i] = (i < len && c < n) ? src[(size_t)i * stride + c] : 0.0f;
    }
  }
}
// rows i of a chunk, columns c0 .. c0 + W - 1 of a row of n, into dst[i][W]; each row times scale[i] if given
template <int W>
__device__ __forceinline__ void stage_rows(const float* src, long long stride, int len, int c0, int n, bool vec, const float* scale,
                                           float* dst) {
  if (vec) {
    for (int x = threadIdx.x; x < SC_Q * (W / 4); x += SC_THREADS) {
      const int i = x / (W / 4), c = x % (W / 4) * 4;
      float4 v = (i < len && c0 + c < n) ? ld4(src + (size_t)i * stride + c0 + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (scale) { const float f = scale[i]; v.x *= f; v.y *= f; v.z *= f; v.w *= f; }
      *reinterpret_cast<float4*>(dst + i * W + c) = v;
    }
  } else {
    for (int x = threadIdx.x; x < SC_Q * W; x += SC_THREADS) {
      const int i = x / W, c = x % W;
      float v = (i < len && c0 + c < n) ? src[(size_t)i * stride + c0 + c] : 0.0f;
      if (scale) v *= scale[i];
      dst[i * W + c] = v;
    }
  }
}
__device__ __forceinline__ void fma16(float (&acc)[4][4], const float4& a, const float4& b) {
  const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
}

// Grid (chunks, H * row tiles + G, column tiles).  Blocks y < H * row tiles: a tile [SC_N x SC_V] of a head's
// contribution; the others (z = 0): a group's products q_i . k_j.
__global__ void __launch_bounds__(SC_THREADS)
chunk_terms_kernel(const ScArgs p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float hi[SC_Q], lo[SC_Q], bs[SC_Q];
  __shared__ Chunk cks;
  pdl_launch_dependents();
  const int c = blockIdx.x, tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  const int row_tiles = (p.N + SC_N - 1) / SC_N;
  const bool products = (int)blockIdx.y >= p.H * row_tiles;
  if (products && blockIdx.z != 0) return;
  const int h = products ? 0 : blockIdx.y / row_tiles, n0 = products ? 0 : blockIdx.y % row_tiles * SC_N, v0 = blockIdx.z * SC_V;
  pdl_wait();
  if (tid < 32) {
    const Chunk ck = find_chunk(p, c);
    if (tid == 0) cks = ck;
    if (!products && ck.r >= 0) chunk_sums(p, h, ck, hi, lo, bs);
  }
  __syncthreads();
  const Chunk ck = cks;
  if (ck.r < 0) return;
  if (products) {
    const int g = blockIdx.y - p.H * row_tiles, np = (p.N + 3) / 4 * 4;
    float* qt = sm;
    float* kt = sm + np * SC_LD;
    stage_columns(p.q + (size_t)ck.t0 * p.q_stride + (size_t)g * p.N, p.q_stride, ck.len, p.N, np, p.vec, qt);
    stage_columns(p.k + (size_t)ck.t0 * p.k_stride + (size_t)g * p.N, p.k_stride, ck.len, p.N, np, p.vec, kt);
    __syncthreads();
    float acc[4][4] = {};
#pragma unroll 4
    for (int n = 0; n < np; n++) fma16(acc, ld4(qt + n * SC_LD + ty * 4), ld4(kt + n * SC_LD + tx * 4));
    float* o = p.qk + ((size_t)c * p.G + g) * SC_Q * SC_Q;
#pragma unroll
    for (int i = 0; i < 4; i++)
      *reinterpret_cast<float4*>(o + (ty * 4 + i) * SC_Q + tx * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    return;
  }
  // k_j v_j^T times exp(c_last - c_j) b_j (taken by v)
  float* ks = sm;
  float* vs = sm + SC_Q * SC_N;
  if (tid < SC_Q) bs[tid] *= expf((hi[ck.len - 1] - hi[tid]) + (lo[ck.len - 1] - lo[tid]));
  if (tid == 0 && n0 == 0 && v0 == 0) p.total[(size_t)c * p.H + h] = expf(hi[ck.len - 1] + lo[ck.len - 1]);
  __syncthreads();
  const int g = h / (p.H / p.G);
  stage_rows<SC_N>(p.k + (size_t)ck.t0 * p.k_stride + (size_t)g * p.N, p.k_stride, ck.len, n0, p.N, p.vec, nullptr, ks);
  stage_rows<SC_V>(p.v + (size_t)ck.t0 * p.v_stride + (size_t)h * p.V, p.v_stride, ck.len, v0, p.V, p.vec, bs, vs);
  __syncthreads();
  const bool two = p.N - n0 > SC_N / 2;       // rows in the tile's second half
  float a0[4][4] = {}, a1[4][4] = {};
  if (two) {
#pragma unroll 4
    for (int j = 0; j < ck.len; j++) {
      const float4 b = ld4(vs + j * SC_V + tx * 4);
      fma16(a0, ld4(ks + j * SC_N + ty * 4), b);
      fma16(a1, ld4(ks + j * SC_N + SC_N / 2 + ty * 4), b);
    }
  } else {
#pragma unroll 4
    for (int j = 0; j < ck.len; j++) fma16(a0, ld4(ks + j * SC_N + ty * 4), ld4(vs + j * SC_V + tx * 4));
  }
  float* o = p.S + ((size_t)c * p.H + h) * p.N * p.V;
  auto write = [&](const float (&a)[4][4], int first) {
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int n = first + i, v = v0 + tx * 4;
      if (n >= p.N) continue;
      if (p.vec) {
        if (v < p.V) *reinterpret_cast<float4*>(o + (size_t)n * p.V + v) = make_float4(a[i][0], a[i][1], a[i][2], a[i][3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; e++)
          if (v + e < p.V) o[(size_t)n * p.V + v + e] = a[i][e];
      }
    }
  };
  write(a0, n0 + ty * 4);
  if (two) write(a1, n0 + SC_N / 2 + ty * 4);
}

// Grid (requests, H, pieces of the state): contributions -> states ahead of the chunks, the last state kept.
constexpr int SC_AHEAD = 4;
template <typename TV>
__global__ void __launch_bounds__(SC_THREADS)
chunk_pass_kernel(const ScArgs p) {
  __shared__ int first_s;
  pdl_launch_dependents();
  const int r = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31;
  pdl_wait();
  if (threadIdx.x < 32) {
    int n = 0;
    for (int x = lane; x < r; x += 32) n += (p.q_start[x + 1] - p.q_start[x] + SC_Q - 1) / SC_Q;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) n += __shfl_xor_sync(0xffffffffu, n, o);
    if (lane == 0) first_s = n;
  }
  __syncthreads();
  const int first = first_s, count = (p.q_start[r + 1] - p.q_start[r] + SC_Q - 1) / SC_Q;
  const int slot = p.state_slots[r];
  if (count <= 0 || !sglc_index_ok(slot, p.n_slots, p.err)) return;
  constexpr int W = sizeof(TV) / 4;
  const long long size = (long long)p.N * p.V / W, i = (long long)blockIdx.z * SC_THREADS + threadIdx.x;
  if (i >= size) return;
  TV* st = reinterpret_cast<TV*>(p.state) + ((size_t)slot * p.H + h) * size + i;
  TV* ch = reinterpret_cast<TV*>(p.S) + ((size_t)first * p.H + h) * size + i;
  const float* d = p.total + (size_t)first * p.H + h;
  const size_t step = (size_t)p.H * size;
  TV s = *st;
  for (int c0 = 0; c0 < count; c0 += SC_AHEAD) {
    TV own[SC_AHEAD];
    float dec[SC_AHEAD];
#pragma unroll
    for (int e = 0; e < SC_AHEAD; e++)
      if (c0 + e < count) {
        own[e] = ch[(c0 + e) * step];
        dec[e] = d[(size_t)(c0 + e) * p.H];
      }
#pragma unroll
    for (int e = 0; e < SC_AHEAD; e++)
      if (c0 + e < count) {
        ch[(c0 + e) * step] = s;
        if constexpr (W == 4) {
          s.x = fmaf(dec[e], s.x, own[e].x); s.y = fmaf(dec[e], s.y, own[e].y);
          s.z = fmaf(dec[e], s.z, own[e].z); s.w = fmaf(dec[e], s.w, own[e].w);
        } else {
          s = fmaf(dec[e], s, own[e]);
        }
      }
  }
  *st = s;
}

// Grid (chunks, H, column tiles): a head's read-outs of a chunk.
__global__ void __launch_bounds__(SC_THREADS)
chunk_read_kernel(const ScArgs p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float hi[SC_Q], lo[SC_Q], bs[SC_Q];
  __shared__ Chunk cks;
  pdl_launch_dependents();
  const int c = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * SC_V, tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  pdl_wait();
  if (tid < 32) {
    const Chunk ck = find_chunk(p, c);
    if (tid == 0) cks = ck;
    if (ck.r >= 0) chunk_sums(p, h, ck, hi, lo, bs);
  }
  __syncthreads();
  const Chunk ck = cks;
  if (ck.r < 0) return;
  const int g = h / (p.H / p.G), np = (p.N + 3) / 4 * 4;
  float* qt = sm;                               // [np][SC_LD]
  float* ss = qt + np * SC_LD;                  // [np][SC_V]
  float* mt = ss + np * SC_V;                   // [SC_Q j][SC_LD i]
  float* vs = mt + SC_Q * SC_LD;                // [SC_Q][SC_V]
  stage_columns(p.q + (size_t)ck.t0 * p.q_stride + (size_t)g * p.N, p.q_stride, ck.len, p.N, np, p.vec, qt);
  stage_rows<SC_V>(p.v + (size_t)ck.t0 * p.v_stride + (size_t)h * p.V, p.v_stride, ck.len, v0, p.V, p.vec, nullptr, vs);
  const float* S = p.S + ((size_t)c * p.H + h) * p.N * p.V;
  if (p.vec) {
    for (int x = tid; x < np * (SC_V / 4); x += SC_THREADS) {
      const int n = x / (SC_V / 4), v = x % (SC_V / 4) * 4;
      *reinterpret_cast<float4*>(ss + n * SC_V + v) =
          (n < p.N && v0 + v < p.V) ? ld4(S + (size_t)n * p.V + v0 + v) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else {
    for (int x = tid; x < np * SC_V; x += SC_THREADS) {
      const int n = x / SC_V, v = x % SC_V;
      ss[x] = (n < p.N && v0 + v < p.V) ? S[(size_t)n * p.V + v0 + v] : 0.0f;
    }
  }
  const float skip = p.skip ? p.skip[h] : 0.0f;
  const float* qk = p.qk + ((size_t)c * p.G + g) * SC_Q * SC_Q;
  for (int x = tid; x < SC_Q * SC_Q / 4; x += SC_THREADS) {      // (a lane a row i, as above)
    const int i = x % SC_Q, j0 = x / SC_Q * 4;
    const float4 w4 = ld4(qk + i * SC_Q + j0);
    const float w[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int j = j0 + e;
      float m = 0.0f;
      if (j <= i && i < ck.len) m = expf((hi[i] - hi[j]) + (lo[i] - lo[j])) * bs[j] * w[e];
      if (j == i) m += skip;
      mt[j * SC_LD + i] = m;
    }
  }
  __syncthreads();
  float acc[4][4] = {};
#pragma unroll 4
  for (int n = 0; n < np; n++) fma16(acc, ld4(qt + n * SC_LD + ty * 4), ld4(ss + n * SC_V + tx * 4));
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const float f = expf(hi[ty * 4 + i] + lo[ty * 4 + i]);
#pragma unroll
    for (int e = 0; e < 4; e++) acc[i][e] *= f;
  }
  const int last = min(ck.len, (tid / 32 + 1) * 8);              // no row of this warp sees a later token
#pragma unroll 4
  for (int j = 0; j < last; j++) fma16(acc, ld4(mt + j * SC_LD + ty * 4), ld4(vs + j * SC_V + tx * 4));
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int t = ty * 4 + i, v = v0 + tx * 4;
    if (t >= ck.len) continue;
    float* o = p.out + (size_t)(ck.t0 + t) * p.out_stride + (size_t)h * p.V + v;
    if (p.vec) {
      if (v < p.V) *reinterpret_cast<float4*>(o) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; e++)
        if (v + e < p.V) o[e] = acc[i][e];
    }
  }
}

SGLC_API int sglc_state_chunk() { return SC_Q; }

// ws: float, n_chunks * (H * N * V + G * SC_Q * SC_Q + H) entries, n_chunks being at least the chunks of the
// step (sum over requests of ceil(tokens / SC_Q)).
SGLC_API int sglc_state_chunks(const float* q, long long q_stride, const float* k, long long k_stride, const float* v,
                               long long v_stride, const float* b, long long b_stride, const float* A_log,
                               const float* skip, float* out, long long out_stride, float* state, int n_slots,
                               const int* q_start, const int* state_slots, int R, int H, int G, int N, int V,
                               float* ws, int n_chunks, int* err, cudaStream_t stream) {
  if (R <= 0 || n_chunks <= 0) return SGLC_OK;
  if (H <= 0 || G <= 0 || H % G != 0 || N <= 0 || V <= 0 || !A_log || !ws) return SGLC_ERR_ARGUMENT;
  const int row_tiles = (N + SC_N - 1) / SC_N, col_tiles = (V + SC_V - 1) / SC_V;
  if (N > SC_MAX_DIM || (long long)H * row_tiles + G > 65535 || col_tiles > 65535) return SGLC_ERR_UNSUPPORTED;
  ScArgs p = {};
  p.q = q; p.q_stride = q_stride; p.k = k; p.k_stride = k_stride; p.v = v; p.v_stride = v_stride; p.b = b; p.b_stride = b_stride;
  p.A_log = A_log; p.skip = skip; p.out = out; p.out_stride = out_stride; p.state = state; p.n_slots = n_slots;
  p.q_start = q_start; p.state_slots = state_slots; p.R = R; p.H = H; p.G = G; p.N = N; p.V = V; p.n_chunks = n_chunks; p.err = err;
  p.qk = ws;                                                     // (first: whole 16-byte pieces whatever the sizes)
  p.S = p.qk + (size_t)n_chunks * G * SC_Q * SC_Q;
  p.total = p.S + (size_t)n_chunks * H * N * V;
  auto al = [](const void* x) { return (reinterpret_cast<uintptr_t>(x) & 15) == 0; };
  if (!al(ws)) return SGLC_ERR_ARGUMENT;
  p.vec = N % 4 == 0 && V % 4 == 0 && (q_stride | k_stride | v_stride | out_stride) % 4 == 0 && al(q) && al(k) && al(v) && al(out);
  const int np = (N + 3) / 4 * 4;
  size_t smem1 = (size_t)SC_Q * (SC_N + SC_V) * 4;
  if ((size_t)2 * np * SC_LD * 4 > smem1) smem1 = (size_t)2 * np * SC_LD * 4;
  const size_t smem3 = ((size_t)np * (SC_LD + SC_V) + SC_Q * (SC_LD + SC_V)) * 4;
  cudaFuncSetAttribute(chunk_terms_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1);
  cudaFuncSetAttribute(chunk_read_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3);
  int rc = sglc_launch(chunk_terms_kernel, dim3(n_chunks, H * row_tiles + G, col_tiles), dim3(SC_THREADS), smem1, stream, 1, true, p);
  if (rc != SGLC_OK) return rc;
  const bool four = ((long long)N * V) % 4 == 0 && al(state);
  const long long pieces = ((long long)N * V / (four ? 4 : 1) + SC_THREADS - 1) / SC_THREADS;
  rc = four ? sglc_launch(chunk_pass_kernel<float4>, dim3(R, H, (unsigned)pieces), dim3(SC_THREADS), 0, stream, 1, true, p)
            : sglc_launch(chunk_pass_kernel<float>, dim3(R, H, (unsigned)pieces), dim3(SC_THREADS), 0, stream, 1, true, p);
  if (rc != SGLC_OK) return rc;
  return sglc_launch(chunk_read_kernel, dim3(n_chunks, H, col_tiles), dim3(SC_THREADS), smem3, stream, 1, true, p);
}

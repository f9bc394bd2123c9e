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
//
// And the same recurrence for steps in which every request brings one token (state_step_kernel): a state is read
// and written once, four columns a thread, all of a thread's rows asked for before the first is worked on.
#include "common.cuh"

SGLC_DEFINE_ERROR_STRING()

constexpr int SC_Q = 64;          // tokens of a chunk
constexpr int SC_V = 64;          // value columns of a tile
constexpr int SC_N = 128;         // state rows of a tile of the contributions
constexpr int SC_PAD = 4;         // floats behind a row of a tile: 16-byte rows, the rows of a warp on different banks
constexpr int SC_LQ = SC_Q + SC_PAD;
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

// The step's chunks in order: request after request, each cut from its own first token.  Called by whole warps.
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
__device__ __forceinline__ void copy16(float* dst, const float* src, bool on) {      // (off: zeros)
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(on ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copies_end_group() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int LEFT>
__device__ __forceinline__ void copies_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory"); }

// rows 0 .. n_rows - 1 of src, columns c0 .. c0 + width - 1 of rows that end at column n, into dst[row][ld]; rows
// from `len` on and columns from n on are zeros.  width is a multiple of 4.
__device__ __forceinline__ void stage(const float* src, long long stride, int n_rows, int len, int c0, int width, int n, bool vec,
                                      float* dst, int ld) {
  if (vec) {
    const int w4 = width / 4;
    for (int x = threadIdx.x; x < n_rows * w4; x += SC_THREADS) {
      const int i = x / w4, c = (x - i * w4) * 4;
      const bool on = i < len && c0 + c < n;
      copy16(dst + i * ld + c, on ? src + (size_t)i * stride + c0 + c : src, on);
    }
  } else {
#pragma unroll 4
    for (int x = threadIdx.x; x < n_rows * width; x += SC_THREADS) {
      const int i = x / width, c = x - i * width;
      dst[i * ld + c] = (i < len && c0 + c < n) ? src[(size_t)i * stride + c0 + c] : 0.0f;
    }
  }
}
// acc[i][j] += a.(row i, entry e) * b[e].(column j), four entries
__device__ __forceinline__ void fma64(float (&acc)[4][4], const float4 (&a)[4], const float4 (&b)[4]) {
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const float av[4] = {a[i].x, a[i].y, a[i].z, a[i].w};
#pragma unroll
    for (int e = 0; e < 4; e++) {
      acc[i][0] = fmaf(av[e], b[e].x, acc[i][0]); acc[i][1] = fmaf(av[e], b[e].y, acc[i][1]);
      acc[i][2] = fmaf(av[e], b[e].z, acc[i][2]); acc[i][3] = fmaf(av[e], b[e].w, acc[i][3]);
    }
  }
}
__device__ __forceinline__ void fma16(float (&acc)[4][4], const float4& a, const float4& b) {
  const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int i = 0; i < 4; i++) {
    acc[i][0] = fmaf(av[i], b.x, acc[i][0]); acc[i][1] = fmaf(av[i], b.y, acc[i][1]);
    acc[i][2] = fmaf(av[i], b.z, acc[i][2]); acc[i][3] = fmaf(av[i], b.w, acc[i][3]);
  }
}
// acc += A rows ty*4 .. +3 (row stride lda) times B (row stride SC_V), over n entries (a multiple of 4)
__device__ __forceinline__ void tile_product(float (&acc)[4][4], const float* A, int lda, const float* B, int n, int ty, int tx) {
  const float* ar = A + ty * 4 * lda;
  const float* br = B + tx * 4;
#pragma unroll 2
  for (int e = 0; e < n; e += 4) {
    float4 a[4], b[4];
#pragma unroll
    for (int i = 0; i < 4; i++) a[i] = ld4(ar + i * lda + e);
#pragma unroll
    for (int i = 0; i < 4; i++) b[i] = ld4(br + (e + i) * SC_V);
    fma64(acc, a, b);
  }
}

// Grid (chunks, H * row tiles + G, column tiles).  Blocks y < H * row tiles: a tile [SC_N x SC_V] of a head's
// contribution; the others (z = 0): a group's products q_i . k_j.
__global__ void __launch_bounds__(SC_THREADS)
chunk_terms_kernel(const ScArgs p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float hi[SC_Q], lo[SC_Q], bs[SC_Q];
  pdl_launch_dependents();
  const int c = blockIdx.x, tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  const int row_tiles = (p.N + SC_N - 1) / SC_N;
  const bool products = (int)blockIdx.y >= p.H * row_tiles;
  const int h = products ? 0 : blockIdx.y / row_tiles, n0 = products ? 0 : blockIdx.y % row_tiles * SC_N, v0 = blockIdx.z * SC_V;
  pdl_wait();
  const Chunk ck = find_chunk(p, c);
  if (ck.r < 0 || (products && blockIdx.z != 0)) return;
  if (products) {
    const int g = blockIdx.y - p.H * row_tiles, np = (p.N + 3) / 4 * 4, ld = np + SC_PAD;
    float* qs = sm;
    float* ks = sm + SC_Q * ld;
    stage(p.q + (size_t)ck.t0 * p.q_stride + (size_t)g * p.N, p.q_stride, SC_Q, ck.len, 0, np, p.N, p.vec, qs, ld);
    stage(p.k + (size_t)ck.t0 * p.k_stride + (size_t)g * p.N, p.k_stride, SC_Q, ck.len, 0, np, p.N, p.vec, ks, ld);
    copies_end_group();
    copies_wait<0>();
    __syncthreads();
    float acc[4][4] = {};
#pragma unroll 2
    for (int e = 0; e < np; e += 4) {                 // (columns j = tx + 16 i: the lanes' rows on different banks)
      float4 a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; i++) a[i] = ld4(qs + (ty * 4 + i) * ld + e);
#pragma unroll
      for (int i = 0; i < 4; i++) b[i] = ld4(ks + (tx + 16 * i) * ld + e);
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
          acc[i][j] = fmaf(a[i].x, b[j].x, acc[i][j]); acc[i][j] = fmaf(a[i].y, b[j].y, acc[i][j]);
          acc[i][j] = fmaf(a[i].z, b[j].z, acc[i][j]); acc[i][j] = fmaf(a[i].w, b[j].w, acc[i][j]);
        }
    }
    float* o = p.qk + ((size_t)c * p.G + g) * SC_Q * SC_Q;
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
      for (int j = 0; j < 4; j++) o[(ty * 4 + i) * SC_Q + tx + 16 * j] = acc[i][j];
    return;
  }
  // k_j v_j^T times exp(c_last - c_j) b_j (taken by v)
  float* ks = sm;
  float* vs = sm + SC_Q * SC_N;
  const int g = h / (p.H / p.G), rows = min(SC_N, (p.N - n0 + 3) / 4 * 4);
  stage(p.v + (size_t)ck.t0 * p.v_stride + (size_t)h * p.V, p.v_stride, SC_Q, ck.len, v0, SC_V, p.V, p.vec, vs, SC_V);
  stage(p.k + (size_t)ck.t0 * p.k_stride + (size_t)g * p.N, p.k_stride, SC_Q, ck.len, n0, rows, p.N, p.vec, ks, SC_N);
  copies_end_group();
  if (tid < 32) chunk_sums(p, h, ck, hi, lo, bs);
  copies_wait<0>();
  __syncthreads();
  if (tid == 0 && n0 == 0 && v0 == 0) p.total[(size_t)c * p.H + h] = expf(hi[ck.len - 1] + lo[ck.len - 1]);
  for (int x = tid; x < SC_Q * SC_V / 4; x += SC_THREADS) {
    const int j = x / (SC_V / 4);
    const float f = bs[j] * expf((hi[ck.len - 1] - hi[j]) + (lo[ck.len - 1] - lo[j]));
    float4 v = ld4(vs + x * 4);
    v.x *= f; v.y *= f; v.z *= f; v.w *= f;
    *reinterpret_cast<float4*>(vs + x * 4) = v;
  }
  __syncthreads();
  const bool two = rows > SC_N / 2;           // rows in the tile's second half
  const bool a_on = ty * 4 < rows, b_on = two && SC_N / 2 + ty * 4 < rows;    // (no row of this thread: nothing to do)
  float a0[4][4] = {}, a1[4][4] = {};
  if (b_on) {
#pragma unroll 4
    for (int j = 0; j < ck.len; j++) {
      const float4 b = ld4(vs + j * SC_V + tx * 4);
      fma16(a0, ld4(ks + j * SC_N + ty * 4), b);
      fma16(a1, ld4(ks + j * SC_N + SC_N / 2 + ty * 4), b);
    }
  } else if (a_on) {
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
  if (a_on) write(a0, n0 + ty * 4);
  if (b_on) write(a1, n0 + SC_N / 2 + ty * 4);
}

// Grid (requests, H, pieces of the state): contributions -> states ahead of the chunks, the last state kept.
constexpr int SC_AHEAD = 8;      // chunks whose contributions are asked for together
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
  pdl_launch_dependents();
  const int c = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * SC_V, tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  pdl_wait();
  const Chunk ck = find_chunk(p, c);
  if (ck.r < 0) return;
  const int g = h / (p.H / p.G), np = (p.N + 3) / 4 * 4, ld = np + SC_PAD;
  float* qs = sm;                               // [SC_Q][ld]
  float* ss = qs + SC_Q * ld;                   // [np][SC_V]
  float* ms = ss + np * SC_V;                   // [SC_Q i][SC_LQ j]
  float* vs = ms + SC_Q * SC_LQ;                // [SC_Q][SC_V]
  stage(p.q + (size_t)ck.t0 * p.q_stride + (size_t)g * p.N, p.q_stride, SC_Q, ck.len, 0, np, p.N, p.vec, qs, ld);
  stage(p.S + ((size_t)c * p.H + h) * p.N * p.V, p.V, np, p.N, v0, SC_V, p.V, p.vec, ss, SC_V);
  copies_end_group();
  stage(p.qk + ((size_t)c * p.G + g) * SC_Q * SC_Q, SC_Q, SC_Q, SC_Q, 0, SC_Q, SC_Q, true, ms, SC_LQ);
  stage(p.v + (size_t)ck.t0 * p.v_stride + (size_t)h * p.V, p.v_stride, SC_Q, ck.len, v0, SC_V, p.V, p.vec, vs, SC_V);
  copies_end_group();
  if (tid < 32) chunk_sums(p, h, ck, hi, lo, bs);
  copies_wait<1>();
  __syncthreads();
  float acc[4][4] = {};
  tile_product(acc, qs, ld, ss, np, ty, tx);
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const float f = expf(hi[ty * 4 + i] + lo[ty * 4 + i]);
#pragma unroll
    for (int e = 0; e < 4; e++) acc[i][e] *= f;
  }
  copies_wait<0>();
  __syncthreads();
  const float skip = p.skip ? p.skip[h] : 0.0f;
  for (int x = tid; x < SC_Q * SC_Q; x += SC_THREADS) {
    const int i = x / SC_Q, j = x % SC_Q;
    float m = 0.0f;
    if (j <= i && i < ck.len) m = expf((hi[i] - hi[j]) + (lo[i] - lo[j])) * bs[j] * ms[i * SC_LQ + j];
    if (j == i) m += skip;
    ms[i * SC_LQ + j] = m;
  }
  __syncthreads();
  tile_product(acc, ms, SC_LQ, vs, (tid / 32 + 1) * 8, ty, tx);        // (no row of this warp sees a later token)
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
  if ((size_t)2 * SC_Q * (np + SC_PAD) * 4 > smem1) smem1 = (size_t)2 * SC_Q * (np + SC_PAD) * 4;
  const size_t smem3 = ((size_t)SC_Q * (np + SC_PAD) + (size_t)np * SC_V + SC_Q * (SC_LQ + SC_V)) * 4;
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

// Every request brings one token (token r is request r's).  Grid (requests, H, column tiles of SS_COLS); a
// thread keeps W columns of every SS_ROWS-th row.
constexpr int SS_COLS = 64, SS_DEEP = 8;
template <int W>      // 4: rows 16 bytes at a time; 1: any sizes
__global__ void __launch_bounds__(SC_THREADS)
state_step_kernel(const ScArgs p, const float* __restrict__ decay, long long decay_stride) {
  constexpr int CT = SS_COLS / W, ROWS = SC_THREADS / CT;        // threads over the columns, rows side by side
  __shared__ float part[ROWS][SS_COLS];
  __shared__ float ks[SC_MAX_DIM], qs[SC_MAX_DIM];
  pdl_launch_dependents();
  const int r = blockIdx.x, h = blockIdx.y, g = h / (p.H / p.G), tid = threadIdx.x;
  const int cx = tid % CT, rx = tid / CT, col = blockIdx.z * SS_COLS + cx * W;
  const bool on = col < p.V;
  const int slot = p.state_slots[r];                             // (nothing a kernel of the step writes)
  if (!sglc_index_ok(slot, p.n_slots, p.err)) return;
  float* st = p.state + ((size_t)slot * p.H + h) * p.N * p.V + col;
  pdl_wait();
  for (int n = tid; n < p.N; n += SC_THREADS) {
    ks[n] = p.k[(size_t)r * p.k_stride + (size_t)g * p.N + n];
    qs[n] = p.q[(size_t)r * p.q_stride + (size_t)g * p.N + n];
  }
  const float b = p.b[(size_t)r * p.b_stride + h], gd = decay[(size_t)r * decay_stride + h];
  float v[W], bv[W], acc[W];
#pragma unroll
  for (int e = 0; e < W; e++) {
    v[e] = on ? p.v[(size_t)r * p.v_stride + (size_t)h * p.V + col + e] : 0.0f;
    bv[e] = b * v[e];
    acc[e] = 0.0f;
  }
  __syncthreads();
  for (int n0 = rx; n0 < p.N; n0 += ROWS * SS_DEEP) {
    float S[SS_DEEP][W];
#pragma unroll
    for (int d = 0; d < SS_DEEP; d++) {
      const int n = n0 + d * ROWS;
      if (on && n < p.N) {
        if constexpr (W == 4) {
          const float4 s = ld4(st + (size_t)n * p.V);
          S[d][0] = s.x; S[d][1] = s.y; S[d][2] = s.z; S[d][3] = s.w;
        } else {
          S[d][0] = st[(size_t)n * p.V];
        }
      }
    }
#pragma unroll
    for (int d = 0; d < SS_DEEP; d++) {
      const int n = n0 + d * ROWS;
      if (on && n < p.N) {
        const float k = ks[n], q = qs[n];
#pragma unroll
        for (int e = 0; e < W; e++) {
          S[d][e] = fmaf(k, bv[e], gd * S[d][e]);
          acc[e] = fmaf(q, S[d][e], acc[e]);
        }
        if constexpr (W == 4) *reinterpret_cast<float4*>(st + (size_t)n * p.V) = make_float4(S[d][0], S[d][1], S[d][2], S[d][3]);
        else st[(size_t)n * p.V] = S[d][0];
      }
    }
  }
#pragma unroll
  for (int e = 0; e < W; e++) part[rx][cx * W + e] = acc[e];
  __syncthreads();
  const int c = blockIdx.z * SS_COLS + tid;
  if (tid < SS_COLS && c < p.V) {
    float o = 0.0f;
#pragma unroll
    for (int x = 0; x < ROWS; x++) o += part[x][tid];
    if (p.skip) o = fmaf(p.skip[h], p.v[(size_t)r * p.v_stride + (size_t)h * p.V + c], o);
    p.out[(size_t)r * p.out_stride + (size_t)h * p.V + c] = o;
  }
}

// S <- decay S + b k v^T, o = S^T q + skip v for R requests of one token each; b and decay: float rows, head h in column h.
SGLC_API int sglc_state_step(const float* q, long long q_stride, const float* k, long long k_stride, const float* v,
                             long long v_stride, const float* b, const float* decay, long long gates_stride,
                             const float* skip, float* out, long long out_stride, float* state, int n_slots,
                             const int* state_slots, int R, int H, int G, int N, int V, int* err, cudaStream_t stream) {
  if (R <= 0) return SGLC_OK;
  if (H <= 0 || G <= 0 || H % G != 0 || N <= 0 || V <= 0 || !b || !decay) return SGLC_ERR_ARGUMENT;
  const int tiles = (V + SS_COLS - 1) / SS_COLS;
  if (N > SC_MAX_DIM || H > 65535 || tiles > 65535) return SGLC_ERR_UNSUPPORTED;
  ScArgs p = {};
  p.q = q; p.q_stride = q_stride; p.k = k; p.k_stride = k_stride; p.v = v; p.v_stride = v_stride; p.b = b; p.b_stride = gates_stride;
  p.skip = skip; p.out = out; p.out_stride = out_stride; p.state = state; p.n_slots = n_slots; p.state_slots = state_slots;
  p.R = R; p.H = H; p.G = G; p.N = N; p.V = V; p.err = err;
  const dim3 grid(R, H, tiles);
  if (V % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0)
    return sglc_launch(state_step_kernel<4>, grid, dim3(SC_THREADS), 0, stream, 1, true, p, decay, gates_stride);
  return sglc_launch(state_step_kernel<1>, grid, dim3(SC_THREADS), 0, stream, 1, true, p, decay, gates_stride);
}

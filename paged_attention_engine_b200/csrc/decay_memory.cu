// A memory that decays: linear attention over a matrix state per head, without softmax or
// denominator. Per token t, with a key k and a query q of n channels (shared by heads / groups
// neighbouring heads), a value v of dv channels, a decay a and a step w per head:
//
//   S <- a_t S + (w_t k_t) v_t^T,        o_t = S^T q_t  (+ skip v_t)
//
// a is exp(log_decay[t, h]) or a constant of the head, w is step[t, h] or one constant. The
// retention of a fixed decay per head and Mamba-2's selective state space are both this
// recurrence. The state is float32 [n][dv] per request and head, carried from token to token.
//
// For float32 operands the arithmetic of `scan` and `step` is double: a read-out sums n products of a
// state that itself sums a thousand tokens, and where the sum cancels, the norm that follows
// multiplies what float32 sums would have lost. The state between two calls is float32 always.
//
// Three ways through it, which give the same numbers up to rounding:
//
//   scan     token after token, any sizes up to 1,024 key channels, float32 or bfloat16 operands. A
//            column of S lives in the registers of KS threads of one warp, a part of its key
//            channels each, so a token costs no barrier.
//   step     requests that bring ONE token: a block per (request, head, range of value columns) reads
//            its part of the state in 16-byte pieces, all of them asked for before the kernel
//            before this one has ended (the state was written in an earlier step), and writes it back.
//   chunked  portions of prompts, bfloat16 operands, in chunks of 128 tokens on tensor cores. With
//            c_i = the sum of log a up to and with token i of the chunk:
//              states  U = sum_j exp(c_last - c_j) w_j k_j v_j^T per chunk, all chunks at once
//              pass    S <- exp(c_last) S + U from chunk to chunk (element-wise)
//              output  o_i = exp(c_i) S_before^T q_i + sum_{j <= i} exp(c_i - c_j) w_j (q_i . k_j) v_j
//            The operands that are products of 32-bit numbers (weighted values, S, weighted scores)
//            go to the tensor core as the sum of two bfloat16 numbers each, so nothing of the
//            recurrence is cut to 16 bits; everything is accumulated in float32.
#include "attention_mma.cuh"

using namespace pae;
using namespace pae_attention;

namespace {

struct Memory {
  const void* q;             // [tokens, q_ld]: group g's channels from g * n
  const void* k;             // [tokens, k_ld]: likewise
  const void* v;             // [tokens, v_ld]: head h's channels from h * dv
  const float* log_decay;    // [tokens, heads], or null: head_decay
  const float* head_decay;   // [heads]
  const float* step;         // [tokens, heads], or null: k_scale
  const float* skip;         // [heads] or null
  float* o;                  // [tokens, heads, dv]
  float* state;              // slot s, head h: state + s * slot_stride + h * n * dv
  const int* q_start;        // [entries + 1]
  const int* state_slot;     // [entries]
  const int* list;           // entries to look at (null: 0, 1, ...)
  long long slot_stride;
  int q_ld, k_ld, v_ld;
  int heads, groups, n, dv;
  int skip_single;           // entries of one token are another kernel's
  float k_scale;
  // chunked
  float* chunk_state;        // [chunk slots, heads, n, dv]
  __nv_bfloat16* before;     // [chunk slots, heads, 2, n, dv]: the state before the chunk, as a sum of two
  float* chunk_decay;        // [chunk slots, heads]
};

// ---------------------------------------------------------------------------------------
// scan
// ---------------------------------------------------------------------------------------
constexpr int SCAN_WARPS = 4;

// The type in which a recurrence over operands of type T is carried within a call.
template <typename T>
struct Carried {
  using type = double;
};
template <>
struct Carried<__nv_bfloat16> {
  using type = float;
};
__device__ __forceinline__ float exp_of(float x) { return expf(x); }
__device__ __forceinline__ double exp_of(double x) { return exp(x); }

template <typename T, int PER, int KS>
__global__ void __launch_bounds__(SCAN_WARPS * 32) memory_scan_kernel(const Memory p) {
  dependent_launch_prologue();
  using A = typename Carried<T>::type;
  constexpr int TILE = KS >= 16 ? 4 : 16;    // tokens at a time in shared memory
  constexpr int SEG = PER + 4;               // a part's channels in shared memory, padded against bank conflicts
  constexpr int ROW = KS * SEG;
  constexpr int WARP_COLS = 32 / KS, COLS = SCAN_WARPS * WARP_COLS;
  __shared__ __align__(16) float qs[TILE][ROW];
  __shared__ __align__(16) float ks[TILE][ROW];
  __shared__ float vs[TILE][COLS], add[TILE];
  __shared__ A keep[TILE];
  const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * COLS;
  const int first = p.q_start[b], count = p.q_start[b + 1] - first;
  if (count <= 0 || (p.skip_single && count == 1)) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, threads = blockDim.x;
  const int g = h / (p.heads / p.groups), n = p.n, dv = p.dv;
  const int part = lane / WARP_COLS, local = warp * WARP_COLS + lane % WARP_COLS, col = c0 + local;
  const bool has_col = col < dv;
  float* st = p.state + (size_t)p.state_slot[b] * p.slot_stride + (size_t)h * n * dv;
  A s[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int row = part * PER + i;
    s[i] = has_col && row < n ? (A)st[(size_t)row * dv + col] : (A)0;
  }
  const A skip = p.skip != nullptr ? p.skip[h] : 0.f;
  const A fixed = p.log_decay == nullptr ? p.head_decay[h] : 0.f;
  for (int t0 = 0; t0 < count; t0 += TILE) {
    const int tokens = min(TILE, count - t0);
    __syncthreads();
    for (int e = tid; e < tokens * KS * PER; e += threads) {
      const int t = e / (KS * PER), i = e - t * (KS * PER), at = (i / PER) * SEG + i % PER;
      const size_t row = (size_t)(first + t0 + t);
      qs[t][at] = i < n ? to_float(((const T*)p.q)[row * p.q_ld + g * n + i]) : 0.f;
      ks[t][at] = i < n ? to_float(((const T*)p.k)[row * p.k_ld + g * n + i]) : 0.f;
    }
    for (int e = tid; e < tokens * COLS; e += threads) {
      const int t = e / COLS, j = e - t * COLS;
      vs[t][j] = c0 + j < dv ? to_float(((const T*)p.v)[(size_t)(first + t0 + t) * p.v_ld + h * dv + c0 + j]) : 0.f;
    }
    if (tid < tokens) {
      const size_t at = (size_t)(first + t0 + tid) * p.heads + h;
      keep[tid] = p.log_decay != nullptr ? exp_of((A)p.log_decay[at]) : fixed;
      add[tid] = p.step != nullptr ? p.step[at] : p.k_scale;
    }
    __syncthreads();
    for (int t = 0; t < tokens; ++t) {
      const A a = keep[t], value = vs[t][local], av = (A)add[t] * value;
      const float* kp = &ks[t][part * SEG];
      const float* qp = &qs[t][part * SEG];
      A sum[4] = {0, 0, 0, 0};
#pragma unroll
      for (int i = 0; i < PER; i += 4) {
        const float4 k4 = *(const float4*)(kp + i), q4 = *(const float4*)(qp + i);
        s[i] = fma(a, s[i], k4.x * av);
        s[i + 1] = fma(a, s[i + 1], k4.y * av);
        s[i + 2] = fma(a, s[i + 2], k4.z * av);
        s[i + 3] = fma(a, s[i + 3], k4.w * av);
        sum[0] = fma(s[i], (A)q4.x, sum[0]);
        sum[1] = fma(s[i + 1], (A)q4.y, sum[1]);
        sum[2] = fma(s[i + 2], (A)q4.z, sum[2]);
        sum[3] = fma(s[i + 3], (A)q4.w, sum[3]);
      }
      A total = (sum[0] + sum[1]) + (sum[2] + sum[3]);
#pragma unroll
      for (int o = WARP_COLS; o < 32; o <<= 1) total += __shfl_xor_sync(0xffffffffu, total, o);
      if (has_col && part == 0) p.o[((size_t)(first + t0 + t) * p.heads + h) * dv + col] = (float)fma(skip, value, total);
    }
  }
  if (has_col) {
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int row = part * PER + i;
      if (row < n) st[(size_t)row * dv + col] = (float)s[i];
    }
  }
}

template <typename T, int PER, int KS>
int launch_scan(const Memory& p, int entries, cudaStream_t s) {
  constexpr int COLS = SCAN_WARPS * (32 / KS);
  launch_kernel(memory_scan_kernel<T, PER, KS>, dim3((p.dv + COLS - 1) / COLS, p.heads, entries), SCAN_WARPS * 32, 0, s, p);
  return check_launch("decay_memory_scan");
}

template <typename T>
int scan_of(const Memory& p, int entries, cudaStream_t s) {
  const int n = p.n;
  if (n <= 16) return launch_scan<T, 4, 4>(p, entries, s);
  if (n <= 32) return launch_scan<T, 8, 4>(p, entries, s);
  if (n <= 48) return launch_scan<T, 12, 4>(p, entries, s);
  if (n <= 64) return launch_scan<T, 16, 4>(p, entries, s);
  if (n <= 96) return launch_scan<T, 24, 4>(p, entries, s);
  if (n <= 128) return launch_scan<T, 32, 4>(p, entries, s);
  if (n <= 256) return launch_scan<T, 32, 8>(p, entries, s);
  if (n <= 512) return launch_scan<T, 32, 16>(p, entries, s);
  return launch_scan<T, 32, 32>(p, entries, s);
}

// ---------------------------------------------------------------------------------------
// step
// ---------------------------------------------------------------------------------------
constexpr int STEP_THREADS = 256;
constexpr int STEP_AHEAD = 8;          // 16-byte pieces of the state that a thread has in flight

template <typename T, int CT>          // CT: value columns of a block
__global__ void __launch_bounds__(STEP_THREADS) memory_step_kernel(const Memory p) {
  using A = typename Carried<T>::type;
  constexpr int CG = CT / 4, LANES = STEP_THREADS / CG;
  extern __shared__ float smem[];      // q [n], k [n]
  __shared__ A sums[STEP_THREADS / 32][CT];
  dependent_launch_trigger();
  const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * CT;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n = p.n, dv = p.dv;
  // The step's integers and the state were written before this step's first kernel was launched.
  const int first = p.q_start[b], count = p.q_start[b + 1] - first;
  const int c = c0 + (tid % CG) * 4, r0 = tid / CG;
  float* st = p.state + (size_t)p.state_slot[b] * p.slot_stride + (size_t)h * n * dv;
  const bool mine = count == 1 && c < dv;
  float4 s[STEP_AHEAD];
#pragma unroll
  for (int i = 0; i < STEP_AHEAD; ++i) {
    const int row = r0 + i * LANES;
    s[i] = mine && row < n ? *(const float4*)(st + (size_t)row * dv + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  dependent_launch_wait();
  if (count != 1) return;
  const int g = h / (p.heads / p.groups);
  const size_t at = (size_t)first * p.heads + h;
  const A w = p.step != nullptr ? p.step[at] : p.k_scale;
  const A a = p.log_decay != nullptr ? exp_of((A)p.log_decay[at]) : (A)p.head_decay[h];
  float* qs = smem;
  float* ks = smem + n;
  for (int i = tid; i < n; i += STEP_THREADS) {
    qs[i] = to_float(((const T*)p.q)[(size_t)first * p.q_ld + g * n + i]);
    ks[i] = to_float(((const T*)p.k)[(size_t)first * p.k_ld + g * n + i]);
  }
  A v[4] = {0, 0, 0, 0};               // the step times the value
  if (mine)
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = w * (A)to_float(((const T*)p.v)[(size_t)first * p.v_ld + h * dv + c + j]);
  __syncthreads();
  A y[4] = {0, 0, 0, 0};
  for (int base = 0; base < n; base += STEP_AHEAD * LANES) {
    if (base > 0) {
#pragma unroll
      for (int i = 0; i < STEP_AHEAD; ++i) {
        const int row = base + r0 + i * LANES;
        if (mine && row < n) s[i] = *(const float4*)(st + (size_t)row * dv + c);
      }
    }
#pragma unroll
    for (int i = 0; i < STEP_AHEAD; ++i) {
      const int row = base + r0 + i * LANES;
      if (!mine || row >= n) continue;
      const A k = ks[row], q = qs[row];
      const A s0 = fma(a, (A)s[i].x, k * v[0]), s1 = fma(a, (A)s[i].y, k * v[1]);
      const A s2 = fma(a, (A)s[i].z, k * v[2]), s3 = fma(a, (A)s[i].w, k * v[3]);
      *(float4*)(st + (size_t)row * dv + c) = make_float4((float)s0, (float)s1, (float)s2, (float)s3);
      y[0] = fma(s0, q, y[0]);
      y[1] = fma(s1, q, y[1]);
      y[2] = fma(s2, q, y[2]);
      y[3] = fma(s3, q, y[3]);
    }
  }
#pragma unroll
  for (int o = CG; o < 32; o <<= 1)
#pragma unroll
    for (int j = 0; j < 4; ++j) y[j] += __shfl_xor_sync(0xffffffffu, y[j], o);
  if (lane < CG)
#pragma unroll
    for (int j = 0; j < 4; ++j) sums[warp][lane * 4 + j] = y[j];
  __syncthreads();
  if (tid < CT && c0 + tid < dv) {
    A total = 0;
#pragma unroll
    for (int i = 0; i < STEP_THREADS / 32; ++i) total += sums[i][tid];
    if (p.skip != nullptr) total = fma((A)p.skip[h], (A)to_float(((const T*)p.v)[(size_t)first * p.v_ld + h * dv + c0 + tid]), total);
    p.o[at * dv + c0 + tid] = (float)total;
  }
}

template <typename T>
int step_of(const Memory& p, int entries, cudaStream_t s) {
  const size_t smem = 2 * sizeof(float) * (size_t)p.n;
  if (p.dv <= 32)
    launch_kernel(memory_step_kernel<T, 32>, dim3(1, p.heads, entries), STEP_THREADS, smem, s, p);
  else
    launch_kernel(memory_step_kernel<T, 64>, dim3((p.dv + 63) / 64, p.heads, entries), STEP_THREADS, smem, s, p);
  return check_launch("decay_memory_step");
}

// ---------------------------------------------------------------------------------------
// chunked
// ---------------------------------------------------------------------------------------
constexpr int CHUNK = 128;

// A chunk's place in the scratch arrays: the chunks of list entry i start behind those of the
// entries before it, whatever their lengths.
__device__ __forceinline__ int chunk_slot(int first_token, int i, int chunk) { return first_token / CHUNK + i + chunk; }

// Threads 0..127: cumulative[t] = the sum of log2 a over the chunk's tokens up to and with t (the
// tokens from `count` on add nothing), weight[t] = w_t. Ends with a barrier.
__device__ __forceinline__ void chunk_decays(const Memory& p, size_t token0, int count, int h, float* cumulative, float* weight) {
  __shared__ float warp_total[CHUNK / 32];
  const int t = threadIdx.x;
  float x = 0.f;
  if (t < CHUNK) {
    if (t < count) {
      const size_t at = (token0 + t) * p.heads + h;
      // a decay of 0 keeps nothing: far below the smallest exponent, but a number
      x = p.log_decay != nullptr ? p.log_decay[at] * LOG2E : fmaxf(log2f(p.head_decay[h]), -1.0e6f);
      weight[t] = p.step != nullptr ? p.step[at] : p.k_scale;
    } else {
      weight[t] = 0.f;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float below = __shfl_up_sync(0xffffffffu, x, o);
      if ((t & 31) >= o) x += below;
    }
    if ((t & 31) == 31) warp_total[t >> 5] = x;
  }
  __syncthreads();
  if (t < CHUNK) {
    for (int w = 0; w < (t >> 5); ++w) x += warp_total[w];
    cumulative[t] = x;
  }
  __syncthreads();
}

// One chunk's own contribution to the state: an NT x 64 tile of U per block, a warp 32 x 32 of it (NT 64 or 128
// key channels: the weighted values are split once for all of them).
constexpr int ST_PITCH = 72;            // bfloat16 elements between rows of a 64-wide tile
template <int NT>
__host__ __device__ constexpr size_t states_smem() { return 2 * (size_t)CHUNK * (NT + 8 + 2 * ST_PITCH); }

template <int NT>
__global__ void __launch_bounds__(2 * NT) memory_chunk_states_kernel(const Memory p) {
  dependent_launch_prologue();
  constexpr int THREADS = 2 * NT, K_PITCH = NT + 8, K_PIECES = NT / 8, V_PER = CHUNK * 8 / THREADS;
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float cumulative[CHUNK], weight[CHUNK];
  const int n_tiles = (p.n + NT - 1) / NT, dv_tiles = (p.dv + 63) / 64;
  const int tile = blockIdx.x % (n_tiles * dv_tiles), chunk = blockIdx.x / (n_tiles * dv_tiles);
  const int h = blockIdx.y, i = blockIdx.z, b = p.list != nullptr ? p.list[i] : i;
  const int first = p.q_start[b], all = p.q_start[b + 1] - first;
  const int count = min(CHUNK, all - chunk * CHUNK);
  if (all == 1 || count <= 0) return;
  const int n0 = (tile % n_tiles) * NT, d0 = (tile / n_tiles) * 64;
  const int g = h / (p.heads / p.groups);
  const size_t token0 = (size_t)first + chunk * CHUNK;
  __nv_bfloat16* ks = (__nv_bfloat16*)raw;                  // [CHUNK][K_PITCH]
  __nv_bfloat16* vh = ks + CHUNK * K_PITCH;                 // [CHUNK][ST_PITCH]
  __nv_bfloat16* vl = vh + CHUNK * ST_PITCH;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
#pragma unroll
  for (int e = tid; e < CHUNK * K_PIECES; e += THREADS) {
    const int row = e / K_PIECES, ch = (e % K_PIECES) * 8;
    __nv_bfloat16* to = ks + row * K_PITCH + ch;
    if (row < count && n0 + ch < p.n)
      cp_async16(smem_u32(to), (const __nv_bfloat16*)p.k + (token0 + row) * p.k_ld + g * p.n + n0 + ch);
    else
      *(uint4*)to = make_uint4(0, 0, 0, 0);
  }
  cp_async_commit();
  uint4 raw_v[V_PER];
#pragma unroll
  for (int j = 0; j < V_PER; ++j) {
    const int e = tid + j * THREADS, row = e >> 3, ch = (e & 7) * 8;
    raw_v[j] = row < count && d0 + ch < p.dv ? *(const uint4*)((const __nv_bfloat16*)p.v + (token0 + row) * p.v_ld + h * p.dv + d0 + ch)
                                             : make_uint4(0, 0, 0, 0);
  }
  chunk_decays(p, token0, count, h, cumulative, weight);
  const float last = cumulative[CHUNK - 1];
  if (tile == 0 && tid == 0) p.chunk_decay[(size_t)chunk_slot(first, i, chunk) * p.heads + h] = exp2f(last);
  if (tid < CHUNK) weight[tid] *= exp2f(last - cumulative[tid]);
  __syncthreads();
#pragma unroll
  for (int j = 0; j < V_PER; ++j) {
    const int e = tid + j * THREADS, row = e >> 3, ch = (e & 7) * 8;
    const float w = weight[row];
    const __nv_bfloat162* v2 = (const __nv_bfloat162*)&raw_v[j];
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float2 f = __bfloat1622float2(v2[u]);
      split_pair(w * f.x, w * f.y, hi[u], lo[u]);
    }
    *(uint4*)(vh + row * ST_PITCH + ch) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *(uint4*)(vl + row * ST_PITCH + ch) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  cp_async_wait<0>();
  __syncthreads();
  const int wn = (warp >> 1) * 32, wd = (warp & 1) * 32;       // the warp's corner of the tile
  if (n0 + wn >= p.n || d0 + wd >= p.dv) return;
  const int mid = lane >> 3, r = lane & 7;
  float acc[2][4][4];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[m][j][0] = acc[m][j][1] = acc[m][j][2] = acc[m][j][3] = 0.f;
  const int steps = (count + 15) / 16;
#pragma unroll 2
  for (int t = 0; t < steps; ++t) {
    uint32_t a[2][4], hi[2][4], lo[2][4];
#pragma unroll
    for (int m = 0; m < 2; ++m)          // rows: key channels, columns: tokens
      ldmatrix_x4_trans(a[m], smem_u32(ks + (t * 16 + (mid >> 1) * 8 + r) * K_PITCH + wn + m * 16 + (mid & 1) * 8));
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int at = (t * 16 + (mid & 1) * 8 + r) * ST_PITCH + wd + j * 16 + (mid >> 1) * 8;
      ldmatrix_x4_trans(hi[j], smem_u32(vh + at));
      ldmatrix_x4_trans(lo[j], smem_u32(vl + at));
    }
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        mma_16816(acc[m][2 * j], a[m], hi[j][0], hi[j][1]);
        mma_16816(acc[m][2 * j + 1], a[m], hi[j][2], hi[j][3]);
      }
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        mma_16816(acc[m][2 * j], a[m], lo[j][0], lo[j][1]);
        mma_16816(acc[m][2 * j + 1], a[m], lo[j][2], lo[j][3]);
      }
  }
  float* out = p.chunk_state + ((size_t)chunk_slot(first, i, chunk) * p.heads + h) * p.n * p.dv;
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = n0 + wn + m * 16 + (lane >> 2) + half * 8;
      if (row >= p.n) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int col = d0 + wd + j * 8 + (lane & 3) * 2;
        if (col < p.dv) *(float2*)(out + (size_t)row * p.dv + col) = make_float2(acc[m][j][half * 2], acc[m][j][half * 2 + 1]);
      }
    }
}

// From chunk to chunk: the state before each (as two bfloat16 planes), and the new state. Four
// neighbouring elements a thread; the contributions of PASS_AHEAD chunks are in flight at a time.
constexpr int PASS_AHEAD = 8;
__global__ void __launch_bounds__(256) memory_chunk_pass_kernel(const Memory p) {
  dependent_launch_prologue();
  const int h = blockIdx.y, i = blockIdx.z, b = p.list != nullptr ? p.list[i] : i;
  const int first = p.q_start[b], count = p.q_start[b + 1] - first;
  const size_t size = (size_t)p.n * p.dv, e = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (count <= 1 || e >= size) return;
  const int chunks = (count + CHUNK - 1) / CHUNK, slot0 = chunk_slot(first, i, 0);
  float* st = p.state + (size_t)p.state_slot[b] * p.slot_stride + (size_t)h * size + e;
  float4 s = *(const float4*)st;
  for (int c0 = 0; c0 < chunks; c0 += PASS_AHEAD) {
    float4 u[PASS_AHEAD];
    float a[PASS_AHEAD];
#pragma unroll
    for (int j = 0; j < PASS_AHEAD; ++j) {
      const int c = c0 + j < chunks ? c0 + j : chunks - 1;
      const size_t at = (size_t)(slot0 + c) * p.heads + h;
      u[j] = *(const float4*)(p.chunk_state + at * size + e);
      a[j] = p.chunk_decay[at];
    }
#pragma unroll
    for (int j = 0; j < PASS_AHEAD; ++j) {
      if (c0 + j >= chunks) break;
      __nv_bfloat16* to = p.before + ((size_t)(slot0 + c0 + j) * p.heads + h) * 2 * size + e;
      uint2 hi, lo;
      split_pair(s.x, s.y, hi.x, lo.x);
      split_pair(s.z, s.w, hi.y, lo.y);
      *(uint2*)to = hi;
      *(uint2*)(to + size) = lo;
      s.x = fmaf(a[j], s.x, u[j].x);
      s.y = fmaf(a[j], s.y, u[j].y);
      s.z = fmaf(a[j], s.z, u[j].z);
      s.w = fmaf(a[j], s.w, u[j].w);
    }
  }
  *(float4*)st = s;
}

// The read-outs of a chunk: eight warps of 16 tokens each, DVT value columns a block. Shared memory: q
// [128], region A: S as two planes, then keys and values of tokens 64..127; region B: keys and values
// of tokens 0..63. Rows are padded by 8 elements.
__host__ __device__ inline size_t output_region_a(int np, int dvt) {
  const size_t s = (size_t)2 * np * (dvt + 8), kv = (size_t)64 * (np + 8) + (size_t)64 * (dvt + 8);
  return s > kv ? s : kv;
}
__host__ __device__ inline size_t output_smem(int np, int dvt) {
  return 2 * ((size_t)CHUNK * (np + 8) + output_region_a(np, dvt) + (size_t)64 * (np + 8) + (size_t)64 * (dvt + 8));
}

constexpr size_t OUTPUT_SMEM_MOST = 220 * 1024;      // beside a kilobyte of static shared memory

template <int DVT>
__global__ void __launch_bounds__(256) memory_chunk_output_kernel(const Memory p) {
  dependent_launch_prologue();
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ __align__(16) float cumulative[CHUNK], weight[CHUNK];
  const int dv_tiles = (p.dv + DVT - 1) / DVT;
  const int d0 = (blockIdx.x % dv_tiles) * DVT, chunk = blockIdx.x / dv_tiles;
  const int h = blockIdx.y, i = blockIdx.z, b = p.list != nullptr ? p.list[i] : i;
  const int first = p.q_start[b], all = p.q_start[b + 1] - first;
  const int count = min(CHUNK, all - chunk * CHUNK);
  if (all == 1 || count <= 0) return;
  const int g = h / (p.heads / p.groups), n = p.n, np = (n + 15) & ~15;
  const int kp = np + 8;
  constexpr int VP = DVT + 8;
  const size_t token0 = (size_t)first + chunk * CHUNK;
  __nv_bfloat16* qs = (__nv_bfloat16*)raw;                 // [CHUNK][kp]
  __nv_bfloat16* region_a = qs + (size_t)CHUNK * kp;
  __nv_bfloat16* sh = region_a;                            // [np][VP]
  __nv_bfloat16* sl = sh + (size_t)np * VP;
  __nv_bfloat16* k0 = region_a + output_region_a(np, DVT); // [64][kp]
  __nv_bfloat16* v0 = k0 + (size_t)64 * kp;                // [64][VP]
  __nv_bfloat16* k1 = region_a;
  __nv_bfloat16* v1 = k1 + (size_t)64 * kp;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  auto fetch_rows = [&](__nv_bfloat16* to, int pitch, const __nv_bfloat16* from, size_t ld, int rows, int limit, int cols, int valid_cols) {
    // a thread keeps its column and steps through the rows (cols <= 2048)
    const int chunks = cols >> 3, stride = 256 / chunks, first_row = tid / chunks, c = (tid - first_row * chunks) * 8;
    if (first_row >= stride) return;
    const bool valid = c < valid_cols;
    __nv_bfloat16* at = to + first_row * pitch + c;
    const __nv_bfloat16* src = from + first_row * ld + c;
    const size_t src_step = stride * ld;
#pragma unroll 4
    for (int row = first_row; row < rows; row += stride) {
      if (valid && row < limit)
        cp_async16(smem_u32(at), src);
      else
        *(uint4*)at = make_uint4(0, 0, 0, 0);
      at += stride * pitch;
      src += src_step;
    }
  };
  const __nv_bfloat16* q_from = (const __nv_bfloat16*)p.q + token0 * p.q_ld + g * n;
  const __nv_bfloat16* k_from = (const __nv_bfloat16*)p.k + token0 * p.k_ld + g * n;
  const __nv_bfloat16* v_from = (const __nv_bfloat16*)p.v + token0 * p.v_ld + h * p.dv + d0;
  const size_t size = (size_t)n * p.dv;
  const __nv_bfloat16* s_from = p.before + ((size_t)chunk_slot(first, i, chunk) * p.heads + h) * 2 * size + d0;
  const int valid_dv = min(DVT, p.dv - d0);
  fetch_rows(qs, kp, q_from, p.q_ld, CHUNK, count, np, n);
  fetch_rows(sh, VP, s_from, p.dv, np, n, DVT, valid_dv);
  fetch_rows(sl, VP, s_from + size, p.dv, np, n, DVT, valid_dv);
  cp_async_commit();
  fetch_rows(k0, kp, k_from, p.k_ld, 64, count, np, n);
  fetch_rows(v0, VP, v_from, p.v_ld, 64, count, DVT, valid_dv);
  cp_async_commit();
  chunk_decays(p, token0, count, h, cumulative, weight);
  cp_async_wait<1>();
  __syncthreads();
  const int row0 = warp * 16, mid = lane >> 3, r = lane & 7;
  const bool live = row0 < count;
  float acc[DVT / 8][4];
#pragma unroll
  for (int j = 0; j < DVT / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  const uint32_t q_at = smem_u32(qs + (size_t)(row0 + (mid & 1) * 8 + r) * kp + (mid >> 1) * 8);
  if (live) {
    for (int t = 0; t < np / 16; ++t) {
      uint32_t a[4], s4[DVT / 16][4];
      ldmatrix_x4(a, q_at + t * 32);
#pragma unroll
      for (int plane = 0; plane < 2; ++plane) {
        const __nv_bfloat16* from = (plane == 0 ? sh : sl) + (t * 16 + (mid & 1) * 8 + r) * VP + (mid >> 1) * 8;
#pragma unroll
        for (int j = 0; j < DVT / 16; ++j) ldmatrix_x4_trans(s4[j], smem_u32(from + j * 16));
#pragma unroll
        for (int j = 0; j < DVT / 16; ++j) {
          mma_16816(acc[2 * j], a, s4[j][0], s4[j][1]);
          mma_16816(acc[2 * j + 1], a, s4[j][2], s4[j][3]);
        }
      }
    }
  }
  __syncthreads();                       // the state's planes are used up: tokens 64..127 take their place
  if (count > 64) {
    fetch_rows(k1, kp, k_from + (size_t)64 * p.k_ld, p.k_ld, 64, count - 64, np, n);
    fetch_rows(v1, VP, v_from + (size_t)64 * p.v_ld, p.v_ld, 64, count - 64, DVT, valid_dv);
  }
  cp_async_commit();
  const int my_row[2] = {row0 + (lane >> 2), row0 + (lane >> 2) + 8};
  const float my_cumulative[2] = {cumulative[my_row[0]], cumulative[my_row[1]]};
  const float from_before[2] = {exp2f(my_cumulative[0]), exp2f(my_cumulative[1])};
#pragma unroll
  for (int j = 0; j < DVT / 8; ++j) {
    acc[j][0] *= from_before[0];
    acc[j][1] *= from_before[0];
    acc[j][2] *= from_before[1];
    acc[j][3] *= from_before[1];
  }
  for (int half = 0; half < 2; ++half) {
    if (half == 0) cp_async_wait<1>(); else cp_async_wait<0>();
    __syncthreads();
    if (!live || row0 < half * 64) continue;
    const __nv_bfloat16* kt = half == 0 ? k0 : k1;
    const __nv_bfloat16* vt = half == 0 ? v0 : v1;
    const int blocks = row0 >= half * 64 + 64 ? 4 : (row0 - half * 64) / 16 + 1;      // 16-token steps that the warp's rows see
    for (int u0 = 0; u0 < blocks; u0 += 2) {           // two of them at a time (the second may be beyond the rows: all masked)
      float s[4][4];
#pragma unroll
      for (int w = 0; w < 4; ++w) s[w][0] = s[w][1] = s[w][2] = s[w][3] = 0.f;
      const uint32_t k_at = smem_u32(kt + (size_t)(u0 * 16 + (mid >> 1) * 8 + r) * kp + (mid & 1) * 8);
      const uint32_t k_next = k_at + 16 * kp * 2;
#pragma unroll 4
      for (int t = 0; t < np / 16; ++t) {
        uint32_t a[4], ka[4], kb[4];
        ldmatrix_x4(a, q_at + t * 32);
        ldmatrix_x4(ka, k_at + t * 32);
        ldmatrix_x4(kb, k_next + t * 32);
        mma_16816(s[0], a, ka[0], ka[1]);
        mma_16816(s[1], a, ka[2], ka[3]);
        mma_16816(s[2], a, kb[0], kb[1]);
        mma_16816(s[3], a, kb[2], kb[3]);
      }
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const int token = half * 64 + u0 * 16 + w * 8 + (lane & 3) * 2;
        const float2 c2 = *(const float2*)(cumulative + token), w2 = *(const float2*)(weight + token);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float c = e & 1 ? c2.y : c2.x, wt = e & 1 ? w2.y : w2.x;
          s[w][e] = token + (e & 1) <= my_row[e >> 1] ? s[w][e] * (wt * fast_exp2(my_cumulative[e >> 1] - c)) : 0.f;
        }
      }
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        if (u0 + x >= blocks) break;
        uint32_t hi[4], lo[4], v4[DVT / 16][4];
#pragma unroll
        for (int j = 0; j < DVT / 16; ++j)
          ldmatrix_x4_trans(v4[j], smem_u32(vt + (size_t)((u0 + x) * 16 + (mid & 1) * 8 + r) * VP + j * 16 + (mid >> 1) * 8));
#pragma unroll
        for (int e = 0; e < 4; ++e) split_pair(s[2 * x + (e >> 1)][(e & 1) * 2], s[2 * x + (e >> 1)][(e & 1) * 2 + 1], hi[e], lo[e]);
#pragma unroll
        for (int j = 0; j < DVT / 16; ++j) {
          mma_16816(acc[2 * j], hi, v4[j][0], v4[j][1]);
          mma_16816(acc[2 * j + 1], hi, v4[j][2], v4[j][3]);
        }
#pragma unroll
        for (int j = 0; j < DVT / 16; ++j) {
          mma_16816(acc[2 * j], lo, v4[j][0], v4[j][1]);
          mma_16816(acc[2 * j + 1], lo, v4[j][2], v4[j][3]);
        }
      }
    }
  }
  if (!live) return;
  const float skip = p.skip != nullptr ? p.skip[h] : 0.f;
  const __nv_bfloat16* own = row0 < 64 ? v0 + (size_t)row0 * VP : v1 + (size_t)(row0 - 64) * VP;      // the warp's tokens' values
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    if (my_row[e] >= count) continue;
    float* out = p.o + ((token0 + my_row[e]) * p.heads + h) * p.dv + d0;
#pragma unroll
    for (int j = 0; j < DVT / 8; ++j) {
      const int col = j * 8 + (lane & 3) * 2;
      if (d0 + col >= p.dv) continue;
      const float2 v2 = __bfloat1622float2(*(const __nv_bfloat162*)(own + (size_t)(my_row[e] - row0) * VP + col));
      *(float2*)(out + col) = make_float2(fmaf(skip, v2.x, acc[j][e * 2]), fmaf(skip, v2.y, acc[j][e * 2 + 1]));
    }
  }
}

int check_memory(const Memory& p, int entries) {
  if (p.heads < 1 || p.groups < 1 || p.heads % p.groups) return fail(2, "decay_memory: %d heads in %d groups", p.heads, p.groups);
  if (p.n < 1 || p.dv < 1 || p.n > 1024) return fail(2, "decay_memory: heads of %d key and %d value channels", p.n, p.dv);
  if (p.log_decay == nullptr && p.head_decay == nullptr) return fail(2, "decay_memory: no decay");
  if (p.heads > 65535 || entries > 65535) return fail(3, "decay_memory: %d heads x %d requests exceed one launch", p.heads, entries);
  return 0;
}

Memory memory_of(float* o, float* state, long long slot_stride, const void* q, int q_ld, const void* k, int k_ld, const void* v,
                 int v_ld, const float* log_decay, const float* head_decay, const float* step, float k_scale, const float* skip,
                 const int* q_start, const int* state_slot, int heads, int groups, int n, int dv) {
  Memory p{};
  p.q = q, p.k = k, p.v = v;
  p.log_decay = log_decay, p.head_decay = head_decay, p.step = step, p.skip = skip;
  p.o = o, p.state = state;
  p.q_start = q_start, p.state_slot = state_slot;
  p.slot_stride = slot_stride;
  p.q_ld = q_ld, p.k_ld = k_ld, p.v_ld = v_ld;
  p.heads = heads, p.groups = groups, p.n = n, p.dv = dv;
  p.k_scale = k_scale;
  return p;
}

int chunk_columns(int n, int dv) {      // value columns of an output block, 0: the sizes do not fit
  const int np = (n + 15) / 16 * 16;
  if (dv > 32 && output_smem(np, 64) <= OUTPUT_SMEM_MOST) return 64;
  return output_smem(np, 32) <= OUTPUT_SMEM_MOST ? 32 : 0;
}

}  // namespace

// Token after token. skip_single: the entries of one token are left to `pae_decay_memory_step`.
PAE_EXPORT int pae_decay_memory_scan(float* o, float* state, long long slot_stride, const void* q, int q_ld, const void* k, int k_ld,
                                     const void* v, int v_ld, const float* log_decay, const float* head_decay, const float* step,
                                     float k_scale, const float* skip, const int* q_start, const int* state_slot, int entries,
                                     int heads, int groups, int n, int dv, int skip_single, int dtype, void* stream) {
  if (entries == 0) return 0;
  Memory p = memory_of(o, state, slot_stride, q, q_ld, k, k_ld, v, v_ld, log_decay, head_decay, step, k_scale, skip, q_start, state_slot,
                       heads, groups, n, dv);
  p.skip_single = skip_single;
  if (int err = check_memory(p, entries)) return err;
  if (dtype == kF32) return scan_of<float>(p, entries, (cudaStream_t)stream);
  if (dtype == kBF16) return scan_of<__nv_bfloat16>(p, entries, (cudaStream_t)stream);
  return fail(1, "decay_memory_scan: unknown dtype %d", dtype);
}

// 1 when the step kernel takes these sizes (16-byte pieces of the state).
PAE_EXPORT int pae_decay_memory_step_supports(int n, int dv, long long slot_stride) {
  return n >= 1 && n <= 1024 && dv % 4 == 0 && slot_stride % 4 == 0 ? 1 : 0;
}

// The entries that bring one token.
PAE_EXPORT int pae_decay_memory_step(float* o, float* state, long long slot_stride, const void* q, int q_ld, const void* k, int k_ld,
                                     const void* v, int v_ld, const float* log_decay, const float* head_decay, const float* step,
                                     float k_scale, const float* skip, const int* q_start, const int* state_slot, int entries,
                                     int heads, int groups, int n, int dv, int dtype, void* stream) {
  if (entries == 0) return 0;
  const Memory p = memory_of(o, state, slot_stride, q, q_ld, k, k_ld, v, v_ld, log_decay, head_decay, step, k_scale, skip, q_start,
                             state_slot, heads, groups, n, dv);
  if (int err = check_memory(p, entries)) return err;
  if (!pae_decay_memory_step_supports(n, dv, slot_stride) || ((uintptr_t)state & 15))
    return fail(2, "decay_memory_step: a state of %d x %d is not made of aligned 16-byte pieces", n, dv);
  if (dtype == kF32) return step_of<float>(p, entries, (cudaStream_t)stream);
  if (dtype == kBF16) return step_of<__nv_bfloat16>(p, entries, (cudaStream_t)stream);
  return fail(1, "decay_memory_step: unknown dtype %d", dtype);
}

// 1 when the chunked kernels take these sizes: rows of 16-byte pieces, and they fit shared memory.
PAE_EXPORT int pae_decay_memory_chunked_supports(int n, int dv, int q_ld, int k_ld, int v_ld, long long slot_stride) {
  return n % 8 == 0 && dv % 8 == 0 && q_ld % 8 == 0 && k_ld % 8 == 0 && v_ld % 8 == 0 && slot_stride % 4 == 0 && chunk_columns(n, dv) > 0;
}

PAE_EXPORT int pae_decay_memory_chunk() { return CHUNK; }

// The entries that bring more than one token, bfloat16. list: `listed` entries to look at (null: all, and
// those of one token are passed over). Scratch for tokens / 128 + listed chunks: chunk_state floats
// [chunks, heads, n, dv], before bfloat16 [chunks, heads, 2, n, dv], chunk_decay floats [chunks, heads]. Three launches.
PAE_EXPORT int pae_decay_memory_chunked(float* o, float* state, long long slot_stride, const void* q, int q_ld, const void* k, int k_ld,
                                        const void* v, int v_ld, const float* log_decay, const float* head_decay, const float* step,
                                        float k_scale, const float* skip, const int* q_start, const int* state_slot, const int* list,
                                        int listed, int max_q_len, int heads, int groups, int n, int dv, float* chunk_state,
                                        void* before, float* chunk_decay, void* stream) {
  if (listed == 0 || max_q_len <= 1) return 0;
  Memory p = memory_of(o, state, slot_stride, q, q_ld, k, k_ld, v, v_ld, log_decay, head_decay, step, k_scale, skip, q_start, state_slot,
                       heads, groups, n, dv);
  p.list = list;
  p.chunk_state = chunk_state, p.before = (__nv_bfloat16*)before, p.chunk_decay = chunk_decay;
  if (int err = check_memory(p, listed)) return err;
  if (!pae_decay_memory_chunked_supports(n, dv, q_ld, k_ld, v_ld, slot_stride))
    return fail(2, "decay_memory_chunked: heads of %d key and %d value channels", n, dv);
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state | (uintptr_t)chunk_state | (uintptr_t)before) & 15)
    return fail(2, "decay_memory_chunked: an operand does not start on a 16-byte boundary");
  cudaStream_t s = (cudaStream_t)stream;
  const int chunks = (max_q_len + CHUNK - 1) / CHUNK;
  if (n > 64) {
    if (int err = allow_smem(memory_chunk_states_kernel<128>, states_smem<128>(), "decay_memory_chunked")) return err;
    launch_kernel(memory_chunk_states_kernel<128>, dim3(chunks * ((n + 127) / 128) * ((dv + 63) / 64), heads, listed), 256, states_smem<128>(), s, p);
  } else {
    if (int err = allow_smem(memory_chunk_states_kernel<64>, states_smem<64>(), "decay_memory_chunked")) return err;
    launch_kernel(memory_chunk_states_kernel<64>, dim3(chunks * ((dv + 63) / 64), heads, listed), 128, states_smem<64>(), s, p);
  }
  if (int err = check_launch("decay_memory_chunk_states")) return err;
  launch_kernel(memory_chunk_pass_kernel, dim3((unsigned)(((size_t)n * dv / 4 + 255) / 256), heads, listed), 256, 0, s, p);
  if (int err = check_launch("decay_memory_chunk_pass")) return err;
  const int columns = chunk_columns(n, dv), np = (n + 15) / 16 * 16;
  const size_t smem = output_smem(np, columns);
  if (columns == 64) {
    if (int err = allow_smem(memory_chunk_output_kernel<64>, OUTPUT_SMEM_MOST, "decay_memory_chunked")) return err;
    launch_kernel(memory_chunk_output_kernel<64>, dim3(chunks * ((dv + 63) / 64), heads, listed), 256, smem, s, p);
  } else {
    if (int err = allow_smem(memory_chunk_output_kernel<32>, OUTPUT_SMEM_MOST, "decay_memory_chunked")) return err;
    launch_kernel(memory_chunk_output_kernel<32>, dim3(chunks * ((dv + 31) / 32), heads, listed), 256, smem, s, p);
  }
  return check_launch("decay_memory_chunk_output");
}

PAE_DEFINE_LAST_ERROR()

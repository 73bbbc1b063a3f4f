// The gated delta rule: a matrix memory per head that forgets by a decay of the token's choice and whose
// write replaces what the memory already holds at the token's key. Per token t, with k and q of n channels
// (shared by heads / groups neighbouring heads), v of dv channels, and per head a decay a and a rate beta:
//
//   k' = k / sqrt(sum k^2 + key_eps)            q' = q_scale q / sqrt(sum q^2 + key_eps)
//   S <- a S;   u = beta (v - S^T k');   S <- S + k' u^T;   o = S^T q'
//
// The state is float32 [n][dv] per request and head, carried from token to token. k and q stay what the
// convolution left (in the engine's element type); their lengths, the decay, beta and the recurrence are
// 32-bit. A unit vector is its raw vector times one number per token, so the raw vectors are the
// operands and the numbers multiply the float32 sums.
//
// Since o = S^T q' reads the state after the write, o = a (S_before^T q') + (k' . q') u: both sums over
// the state run over the old one, side by side.
//
// For float32 operands the arithmetic of `scan` and `step` is double: u is a difference of the value
// and a sum over the state, and where the two nearly cancel, the norm that follows multiplies what
// float32 sums would have lost. The state between two calls is float32 always.
//
// Three ways through it, which give the same numbers up to rounding:
//
//   scan     token after token, any sizes up to 1,024 key channels, float32 or bfloat16 operands. A
//            column of S lives in the registers of KS threads of one warp.
//   step     requests that bring ONE token: a block per (request, head, range of value columns); its part
//            of the state is asked for before the kernel before this one has ended.
//   chunked  portions of prompts, bfloat16 operands, in chunks of 64 tokens on tensor cores (the WY form of
//            Yang, Kautz and Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule"). With
//            c_i = the sum of log a up to and with token i of the chunk, A_ij = beta_i exp(c_i - c_j) (k'_i . k'_j)
//            for j < i (else 0), and S the state before the chunk:
//              solve   (I + A) [U0 | W] = [beta v | beta exp(c) k'] by block substitution, all chunks at once
//              pass    U = U0 - W S;  S <- exp(c_last) S + sum_j exp(c_last - c_j) k'_j u_j^T from chunk to chunk
//              output  o_i = exp(c_i) S^T q'_i + sum_{j <= i} exp(c_i - c_j) (q'_i . k'_j) u_j, all chunks at once
//            What is 32-bit and has to be an operand of a tensor core (A, its solution, W, S, U, weighted
//            scores) goes in as the sum of two bfloat16 numbers, so nothing of the recurrence is cut to 16 bits;
//            everything is accumulated in float32.
#include "attention_mma.cuh"

using namespace pae;
using namespace pae_attention;

namespace {

struct Delta {
  const void* q;             // [tokens, q_ld]: group g's channels from g * n
  const void* k;             // [tokens, k_ld]: likewise
  const void* v;             // [tokens, v_ld]: head h's channels from h * dv
  const float* log_decay;    // [tokens, heads]
  const float* beta;         // [tokens, heads]
  float* o;                  // [tokens, heads, dv]
  float* state;              // slot s, head h: state + s * slot_stride + h * n * dv
  const int* q_start;        // [entries + 1]
  const int* state_slot;     // [entries]
  const int* list;           // entries to look at (null: 0, 1, ...)
  long long slot_stride;
  int q_ld, k_ld, v_ld;
  int heads, groups, n, dv;
  int skip_single;           // entries of one token are another kernel's
  float key_eps, q_scale;
  // chunked, per (chunk slot, head)
  __nv_bfloat16* wk;         // [3, 64, pitch]: W as a sum of two, and K
  float* u0;                 // [dv, 64]
  __nv_bfloat16* u;          // [2, dv, 64]: U as a sum of two
  __nv_bfloat16* before;     // [2, dv, n]: the state before the chunk, as a sum of two
  float* vec;                // [2, 64]: c in units of log 2, and 1 / |k|
};

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
__device__ __forceinline__ float inverse_root(float x) { return 1.f / sqrtf(x); }
__device__ __forceinline__ double inverse_root(double x) { return 1.0 / sqrt(x); }

template <typename A>
__device__ __forceinline__ A all_sum(A v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// ---------------------------------------------------------------------------------------
// scan
// ---------------------------------------------------------------------------------------
constexpr int SCAN_WARPS = 4;

template <typename T, int PER, int KS>
__global__ void __launch_bounds__(SCAN_WARPS * 32) delta_scan_kernel(const Delta p) {
  dependent_launch_prologue();
  using A = typename Carried<T>::type;
  constexpr int TILE = KS >= 16 ? 4 : 16;    // tokens at a time in shared memory
  constexpr int SEG = PER + 4;               // a part's channels in shared memory, padded against bank conflicts
  constexpr int ROW = KS * SEG;
  constexpr int WARP_COLS = 32 / KS, COLS = SCAN_WARPS * WARP_COLS;
  __shared__ __align__(16) float qs[TILE][ROW];
  __shared__ __align__(16) float ks[TILE][ROW];
  __shared__ float vs[TILE][COLS];
  __shared__ A keep[TILE], rate[TILE], k_inv[TILE], q_inv[TILE], kq[TILE];
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
      keep[tid] = exp_of((A)p.log_decay[at]);
      rate[tid] = p.beta[at];
    }
    __syncthreads();
    for (int t = warp; t < tokens; t += SCAN_WARPS) {      // the tile's lengths and k . q, a warp a token
      A kk = 0, qq = 0, both = 0;
      for (int i = lane; i < KS * PER; i += 32) {
        const int at = (i / PER) * SEG + i % PER;
        const A k = ks[t][at], q = qs[t][at];
        kk = fma(k, k, kk);
        qq = fma(q, q, qq);
        both = fma(k, q, both);
      }
      kk = all_sum(kk), qq = all_sum(qq), both = all_sum(both);
      if (lane == 0) {
        k_inv[t] = inverse_root(kk + (A)p.key_eps);
        q_inv[t] = inverse_root(qq + (A)p.key_eps) * (A)p.q_scale;
        kq[t] = both * k_inv[t] * q_inv[t];
      }
    }
    __syncthreads();
    for (int t = 0; t < tokens; ++t) {
      const float* kp = &ks[t][part * SEG];
      const float* qp = &qs[t][part * SEG];
      A sk[2] = {0, 0}, sq[2] = {0, 0};
#pragma unroll
      for (int i = 0; i < PER; i += 4) {
        const float4 k4 = *(const float4*)(kp + i), q4 = *(const float4*)(qp + i);
        sk[0] = fma(s[i], (A)k4.x, sk[0]);
        sq[0] = fma(s[i], (A)q4.x, sq[0]);
        sk[1] = fma(s[i + 1], (A)k4.y, sk[1]);
        sq[1] = fma(s[i + 1], (A)q4.y, sq[1]);
        sk[0] = fma(s[i + 2], (A)k4.z, sk[0]);
        sq[0] = fma(s[i + 2], (A)q4.z, sq[0]);
        sk[1] = fma(s[i + 3], (A)k4.w, sk[1]);
        sq[1] = fma(s[i + 3], (A)q4.w, sq[1]);
      }
      A k_sum = sk[0] + sk[1], q_sum = sq[0] + sq[1];
#pragma unroll
      for (int o = WARP_COLS; o < 32; o <<= 1) {
        k_sum += __shfl_xor_sync(0xffffffffu, k_sum, o);
        q_sum += __shfl_xor_sync(0xffffffffu, q_sum, o);
      }
      const A a = keep[t], u = rate[t] * ((A)vs[t][local] - a * k_inv[t] * k_sum), uk = k_inv[t] * u;
#pragma unroll
      for (int i = 0; i < PER; i += 4) {
        const float4 k4 = *(const float4*)(kp + i);
        s[i] = fma(a, s[i], (A)k4.x * uk);
        s[i + 1] = fma(a, s[i + 1], (A)k4.y * uk);
        s[i + 2] = fma(a, s[i + 2], (A)k4.z * uk);
        s[i + 3] = fma(a, s[i + 3], (A)k4.w * uk);
      }
      if (has_col && part == 0) p.o[((size_t)(first + t0 + t) * p.heads + h) * dv + col] = (float)fma(kq[t], u, a * q_inv[t] * q_sum);
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
int launch_scan(const Delta& p, int entries, cudaStream_t s) {
  constexpr int COLS = SCAN_WARPS * (32 / KS);
  launch_kernel(delta_scan_kernel<T, PER, KS>, dim3((p.dv + COLS - 1) / COLS, p.heads, entries), SCAN_WARPS * 32, 0, s, p);
  return check_launch("gated_delta_scan");
}

template <typename T>
int scan_of(const Delta& p, int entries, cudaStream_t s) {
  const int n = p.n;
  if (n <= 16) return launch_scan<T, 4, 4>(p, entries, s);
  if (n <= 32) return launch_scan<T, 8, 4>(p, entries, s);
  if (n <= 64) return launch_scan<T, 16, 4>(p, entries, s);
  if (n <= 128) return launch_scan<T, 16, 8>(p, entries, s);
  if (n <= 256) return launch_scan<T, 16, 16>(p, entries, s);
  if (n <= 512) return launch_scan<T, 16, 32>(p, entries, s);
  return launch_scan<T, 32, 32>(p, entries, s);
}

// ---------------------------------------------------------------------------------------
// step
// ---------------------------------------------------------------------------------------
constexpr int STEP_THREADS = 256;
constexpr int STEP_AHEAD = 8;          // 16-byte pieces of the state that a thread keeps

template <typename T, int CT>          // CT: value columns of a block
__global__ void __launch_bounds__(STEP_THREADS) delta_step_kernel(const Delta p) {
  using A = typename Carried<T>::type;
  constexpr int CG = CT / 4, LANES = STEP_THREADS / CG, WARPS = STEP_THREADS / 32;
  extern __shared__ float smem[];      // q [n], k [n]
  __shared__ A k_sums[WARPS][CT], q_sums[WARPS][CT];
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
  const A a = exp_of((A)p.log_decay[at]), beta = p.beta[at];
  float* qs = smem;
  float* ks = smem + n;
  for (int i = tid; i < n; i += STEP_THREADS) {
    qs[i] = to_float(((const T*)p.q)[(size_t)first * p.q_ld + g * n + i]);
    ks[i] = to_float(((const T*)p.k)[(size_t)first * p.k_ld + g * n + i]);
  }
  A v[4] = {0, 0, 0, 0};
  if (mine)
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = to_float(((const T*)p.v)[(size_t)first * p.v_ld + h * dv + c + j]);
  __syncthreads();
  A kk = 0, qq = 0, both = 0;            // every warp for itself
  for (int i = lane; i < n; i += 32) {
    const A k = ks[i], q = qs[i];
    kk = fma(k, k, kk);
    qq = fma(q, q, qq);
    both = fma(k, q, both);
  }
  const A k_inv = inverse_root(all_sum(kk) + (A)p.key_eps), q_inv = inverse_root(all_sum(qq) + (A)p.key_eps) * (A)p.q_scale;
  const A kq = all_sum(both) * k_inv * q_inv;
  A sk[4] = {0, 0, 0, 0}, sq[4] = {0, 0, 0, 0};
  auto add = [&](const float4& x, int row) {
    const A k = ks[row], q = qs[row];
    sk[0] = fma((A)x.x, k, sk[0]), sq[0] = fma((A)x.x, q, sq[0]);
    sk[1] = fma((A)x.y, k, sk[1]), sq[1] = fma((A)x.y, q, sq[1]);
    sk[2] = fma((A)x.z, k, sk[2]), sq[2] = fma((A)x.z, q, sq[2]);
    sk[3] = fma((A)x.w, k, sk[3]), sq[3] = fma((A)x.w, q, sq[3]);
  };
  constexpr int HELD = STEP_AHEAD * LANES;       // rows beyond are read twice
#pragma unroll
  for (int i = 0; i < STEP_AHEAD; ++i)
    if (mine && r0 + i * LANES < n) add(s[i], r0 + i * LANES);
  if (mine)
    for (int row = HELD + r0; row < n; row += LANES) add(*(const float4*)(st + (size_t)row * dv + c), row);
#pragma unroll
  for (int o = CG; o < 32; o <<= 1)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      sk[j] += __shfl_xor_sync(0xffffffffu, sk[j], o);
      sq[j] += __shfl_xor_sync(0xffffffffu, sq[j], o);
    }
  if (lane < CG)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      k_sums[warp][lane * 4 + j] = sk[j];
      q_sums[warp][lane * 4 + j] = sq[j];
    }
  __syncthreads();
  A u[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    A total = 0;
#pragma unroll
    for (int i = 0; i < WARPS; ++i) total += k_sums[i][(tid % CG) * 4 + j];
    u[j] = beta * (v[j] - a * k_inv * total);
  }
  if (!mine) return;
  if (r0 == 0) {
    float out[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      A total = 0;
#pragma unroll
      for (int i = 0; i < WARPS; ++i) total += q_sums[i][(tid % CG) * 4 + j];
      out[j] = (float)fma(kq, u[j], a * q_inv * total);
    }
    *(float4*)(p.o + at * dv + c) = make_float4(out[0], out[1], out[2], out[3]);
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) u[j] *= k_inv;
  auto renew = [&](const float4& x, int row) {
    const A k = ks[row];
    *(float4*)(st + (size_t)row * dv + c) =
        make_float4((float)fma(a, (A)x.x, k * u[0]), (float)fma(a, (A)x.y, k * u[1]), (float)fma(a, (A)x.z, k * u[2]), (float)fma(a, (A)x.w, k * u[3]));
  };
#pragma unroll
  for (int i = 0; i < STEP_AHEAD; ++i)
    if (r0 + i * LANES < n) renew(s[i], r0 + i * LANES);
  for (int row = HELD + r0; row < n; row += LANES) renew(*(const float4*)(st + (size_t)row * dv + c), row);
}

template <typename T>
int step_of(const Delta& p, int entries, cudaStream_t s) {
  const size_t smem = 2 * sizeof(float) * (size_t)p.n;
  if (p.dv <= 32 || (long long)entries * p.heads * ((p.dv + 63) / 64) < 148)
    launch_kernel(delta_step_kernel<T, 32>, dim3((p.dv + 31) / 32, p.heads, entries), STEP_THREADS, smem, s, p);
  else
    launch_kernel(delta_step_kernel<T, 64>, dim3((p.dv + 63) / 64, p.heads, entries), STEP_THREADS, smem, s, p);
  return check_launch("gated_delta_step");
}

// ---------------------------------------------------------------------------------------
// chunked: solve
// ---------------------------------------------------------------------------------------
constexpr int CHUNK = 64;
constexpr int A_PITCH = CHUNK + 4;

// A chunk's place in the scratch arrays: the chunks of list entry i start behind those of the
// entries before it, whatever their lengths.
__device__ __forceinline__ int chunk_slot(int first_token, int i, int chunk) { return first_token / CHUNK + i + chunk; }

// rows x cols bfloat16 (cols a multiple of 8) into shared memory by cp.async; rows from `limit` on and
// columns from `valid_cols` on are zeros.
__device__ __forceinline__ void fetch_rows(__nv_bfloat16* to, int pitch, const __nv_bfloat16* from, size_t ld, int rows, int limit, int cols,
                                           int valid_cols) {
  // a thread keeps its column and steps through the rows (cols <= 8 x the block's threads)
  const int pieces = cols >> 3, stride = blockDim.x / pieces, first = threadIdx.x / pieces, c = (threadIdx.x - first * pieces) * 8;
  if (first >= stride) return;
  const bool valid = c < valid_cols;
  __nv_bfloat16* at = to + first * pitch + c;
  const __nv_bfloat16* src = from + first * ld + c;
  const size_t src_step = stride * ld;
#pragma unroll 4
  for (int row = first; row < rows; row += stride) {
    if (valid && row < limit)
      cp_async16(smem_u32(at), src);
    else
      *(uint4*)at = make_uint4(0, 0, 0, 0);
    at += stride * pitch;
    src += src_step;
  }
}

// The squared length of row t of a chunk's keys or queries in shared memory, by four neighbouring threads.
__device__ __forceinline__ float row_squares(const __nv_bfloat16* rows, int pitch, int cols, int t) {
  float sum = 0.f;
  for (int e = (threadIdx.x & 3) * 8; e < cols; e += 32) {
    const uint4 eight = *(const uint4*)(rows + t * pitch + e);
    const __nv_bfloat162* two = (const __nv_bfloat162*)&eight;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 f = __bfloat1622float2(two[j]);
      sum = fmaf(f.x, f.x, fmaf(f.y, f.y, sum));
    }
  }
  sum += __shfl_xor_sync(0xffffffffu, sum, 1);
  return sum + __shfl_xor_sync(0xffffffffu, sum, 2);
}

// Key channels of a chunk's operands in scratch and in the kernels that share them: steps of 32, and a row's
// pitch, padded so that the eight rows of an ldmatrix fall into different banks.
__host__ __device__ inline int padded(int n) { return (n + 31) & ~31; }
__host__ __device__ inline int pitch_of(int n) { return padded(n) + 8; }

__device__ __forceinline__ void stmatrix_x4_trans(uint32_t address, const uint32_t* r) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1, %2, %3, %4};" ::"r"(address), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3])
               : "memory");
}

constexpr int SOLVE_THREADS = 256;
constexpr int L_PITCH = CHUNK + 8;            // of A in shared memory, bfloat16 elements
constexpr int D_PITCH = 24;                   // of the diagonal blocks' inverses
__host__ __device__ inline size_t solve_smem(int n, int dv) {
  const int vp = ((dv + 15) & ~15) + 8;
  return 2 * ((size_t)3 * CHUNK * pitch_of(n) + (size_t)CHUNK * vp + (size_t)2 * CHUNK * L_PITCH + (size_t)2 * CHUNK * D_PITCH);
}

// (I + A) X = B by blocks of 16 rows: Y_r = B_r - sum_{c < r} A_rc X_c, X_r = (I + A_rr)^-1 Y_r. The
// 16 x 16 inverses are float32 forward substitutions; the products run on the tensor cores, every
// operand as the sum of two bfloat16 numbers (three products of four), in the transposed form X^T = ... A^T, whose
// result in registers is the next product's operand as it is. A warp owns 16 columns of X (two sets of them at a
// time) from the first row to the last, so the substitution needs no barrier.
__global__ void __launch_bounds__(SOLVE_THREADS, 2) delta_solve_kernel(const Delta p) {
  dependent_launch_prologue();
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ __align__(16) float cumulative[CHUNK], rate[CHUNK], k_inv[CHUNK], factor_v[CHUNK], factor_k[CHUNK];
  __shared__ float diagonal[CHUNK / 16][16][17];
  const int chunk = blockIdx.x, h = blockIdx.y, i = blockIdx.z, b = p.list != nullptr ? p.list[i] : i;
  const int first = p.q_start[b], all = p.q_start[b + 1] - first;
  const int count = min(CHUNK, all - chunk * CHUNK);
  if (all == 1 || count <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mid = lane >> 3, r = lane & 7;
  const int n = p.n, dv = p.dv, np = padded(n), kp = np + 8, dvp = (dv + 15) & ~15, vp = dvp + 8, g = h / (p.heads / p.groups);
  const size_t token0 = (size_t)first + chunk * CHUNK;
  const size_t unit = (size_t)chunk_slot(first, i, chunk) * p.heads + h;
  __nv_bfloat16* wh = (__nv_bfloat16*)raw;               // [CHUNK][kp]: W, and behind it K, as the pass kernel wants them
  __nv_bfloat16* wl = wh + (size_t)CHUNK * kp;
  __nv_bfloat16* ks = wl + (size_t)CHUNK * kp;
  __nv_bfloat16* vs = ks + (size_t)CHUNK * kp;           // [CHUNK][vp]
  __nv_bfloat16* ah = vs + (size_t)CHUNK * vp;           // [CHUNK][L_PITCH]: A below the diagonal blocks
  __nv_bfloat16* al = ah + (size_t)CHUNK * L_PITCH;
  __nv_bfloat16* th = al + (size_t)CHUNK * L_PITCH;      // [CHUNK][D_PITCH]: (I + A_rr)^-1 - I
  __nv_bfloat16* tl = th + (size_t)CHUNK * D_PITCH;
  fetch_rows(ks, kp, (const __nv_bfloat16*)p.k + token0 * p.k_ld + g * n, p.k_ld, CHUNK, count, np, n);
  cp_async_commit();
  fetch_rows(vs, vp, (const __nv_bfloat16*)p.v + token0 * p.v_ld + h * dv, p.v_ld, CHUNK, count, dvp, dv);
  cp_async_commit();
  if (warp == 0) {                                       // two tokens a lane
    float x[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = lane * 2 + e;
      // far below the smallest float32 exponent a decay keeps nothing: but a number
      x[e] = t < count ? fmaxf(p.log_decay[(token0 + t) * p.heads + h] * LOG2E, -256.f) : 0.f;
      rate[t] = t < count ? p.beta[(token0 + t) * p.heads + h] : 0.f;
    }
    float sum = x[0] + x[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float below = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += below;
    }
    cumulative[lane * 2] = sum - x[1];
    cumulative[lane * 2 + 1] = sum;
  }
  cp_async_wait<1>();
  __syncthreads();
  {
    const int t = tid >> 2;
    const float kk = row_squares(ks, kp, np, t);
    if ((tid & 3) == 0) {
      const float inv = inverse_root(kk + p.key_eps);
      k_inv[t] = inv;
      factor_v[t] = rate[t];
      factor_k[t] = rate[t] * inv * exp2f(cumulative[t]);
      p.vec[unit * 2 * CHUNK + t] = cumulative[t];
      p.vec[unit * 2 * CHUNK + CHUNK + t] = inv;
    }
  }
  __syncthreads();
  {  // A: a warp 16 x 32 of it
    const int row0 = (warp >> 1) * 16, col0 = (warp & 1) * 32;
    if (col0 <= row0 + 15) {
      float acc[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
      const uint32_t a_at = smem_u32(ks + (size_t)(row0 + (mid & 1) * 8 + r) * kp + (mid >> 1) * 8);
      const uint32_t b_at = smem_u32(ks + (size_t)(col0 + (mid >> 1) * 8 + r) * kp + (mid & 1) * 8);
#pragma unroll 4
      for (int t = 0; t < np / 16; ++t) {
        uint32_t a[4], b0[4], b1[4];
        ldmatrix_x4(a, a_at + t * 32);
        ldmatrix_x4(b0, b_at + t * 32);
        ldmatrix_x4(b1, b_at + 16 * kp * 2 + t * 32);
        mma_16816(acc[0], a, b0[0], b0[1]);
        mma_16816(acc[1], a, b0[2], b0[3]);
        mma_16816(acc[2], a, b1[0], b1[1]);
        mma_16816(acc[3], a, b1[2], b1[3]);
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = row0 + (lane >> 2) + half * 8;
        const float at_row = cumulative[row], f = rate[row] * k_inv[row];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int col = col0 + j * 8 + (lane & 3) * 2;
          const float2 c2 = *(const float2*)(cumulative + col), i2 = *(const float2*)(k_inv + col);
          const float x = col < row ? acc[j][half * 2] * (f * i2.x * exp2f(at_row - c2.x)) : 0.f;
          const float y = col + 1 < row ? acc[j][half * 2 + 1] * (f * i2.y * exp2f(at_row - c2.y)) : 0.f;
          if ((col >> 4) == (row >> 4)) {
            diagonal[row >> 4][row & 15][col & 15] = x;
            diagonal[row >> 4][row & 15][(col & 15) + 1] = y;
          } else {
            uint32_t hi, lo;
            split_pair(x, y, hi, lo);
            *(uint32_t*)(ah + row * L_PITCH + col) = hi;
            *(uint32_t*)(al + row * L_PITCH + col) = lo;
          }
        }
      }
    }
  }
  __syncthreads();
  if (warp < CHUNK / 16 && lane < 16) {                  // a column of a diagonal block's inverse a lane
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      float sum = t == lane ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < t; ++j) sum = fmaf(-diagonal[warp][t][j], x[j], sum);
      x[t] = sum;
      const float off = t == lane ? 0.f : sum;
      const __nv_bfloat16 top = __float2bfloat16_rn(off);
      th[(warp * 16 + t) * D_PITCH + lane] = top;
      tl[(warp * 16 + t) * D_PITCH + lane] = __float2bfloat16_rn(off - __bfloat162float(top));
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  // Sets of 16 columns: those of V, then those of K; two sets a warp at a time.
  const int v_sets = dvp / 16, sets = v_sets + np / 16;
  const int own = (mid & 1) * 8, beside = (mid >> 1) * 8;
  for (int s0 = warp; s0 < sets; s0 += 16) {
    uint32_t xh[2][CHUNK / 16][4], xl[2][CHUNK / 16][4];
#pragma unroll
    for (int rb = 0; rb < CHUNK / 16; ++rb) {
      float sum[2][2][4];
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int j = 0; j < 2; ++j) sum[m][j][0] = sum[m][j][1] = sum[m][j][2] = sum[m][j][3] = 0.f;
#pragma unroll
      for (int c = 0; c < rb; ++c) {
        uint32_t bh[4], bl[4];
        const int at = (rb * 16 + beside + r) * L_PITCH + c * 16 + own;
        ldmatrix_x4(bh, smem_u32(ah + at));
        ldmatrix_x4(bl, smem_u32(al + at));
        // the three products of a sum stand four others apart
#pragma unroll
        for (int x = 0; x < 3; ++x)
#pragma unroll
          for (int m = 0; m < 2; ++m)
#pragma unroll
            for (int j = 0; j < 2; ++j)
              mma_16816(sum[m][j], x == 1 ? xl[m][c] : xh[m][c], x == 2 ? bl[2 * j] : bh[2 * j], x == 2 ? bl[2 * j + 1] : bh[2 * j + 1]);
      }
      uint32_t dh[4], dl[4];
      {
        const int at = (rb * 16 + beside + r) * D_PITCH + own;
        ldmatrix_x4(dh, smem_u32(th + at));
        ldmatrix_x4(dl, smem_u32(tl + at));
      }
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const int set = s0 + m * 8;
        if (set >= sets) break;
        const bool is_v = set < v_sets;
        const int col0 = is_v ? set * 16 : (set - v_sets) * 16;
        // element [j][e]: row rb 16 + j 8 + (lane & 3) 2 + (e & 1), column col0 + (lane >> 2) + (e >> 1) 8
        uint32_t raw4[4];
        ldmatrix_x4_trans(raw4, smem_u32((is_v ? vs : ks) + (size_t)(rb * 16 + beside + r) * (is_v ? vp : kp) + col0 + own));
        float y[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const float2 f = *(const float2*)((is_v ? factor_v : factor_k) + rb * 16 + j * 8 + (lane & 3) * 2);
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const float2 two = __bfloat1622float2(*(const __nv_bfloat162*)&raw4[2 * j + half]);
            y[j][half * 2] = fmaf(two.x, f.x, -sum[m][j][half * 2]);
            y[j][half * 2 + 1] = fmaf(two.y, f.y, -sum[m][j][half * 2 + 1]);
          }
        }
        uint32_t yh[4], yl[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split_pair(y[e >> 1][(e & 1) * 2], y[e >> 1][(e & 1) * 2 + 1], yh[e], yl[e]);
#pragma unroll
        for (int x = 0; x < 3; ++x)
#pragma unroll
          for (int j = 0; j < 2; ++j)
            mma_16816(y[j], x == 1 ? yl : yh, x == 2 ? dl[2 * j] : dh[2 * j], x == 2 ? dl[2 * j + 1] : dh[2 * j + 1]);
#pragma unroll
        for (int e = 0; e < 4; ++e) split_pair(y[e >> 1][(e & 1) * 2], y[e >> 1][(e & 1) * 2 + 1], xh[m][rb][e], xl[m][rb][e]);
        if (is_v) {
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int col = col0 + (lane >> 2) + half * 8;
            if (col >= dv) continue;
            float* to = p.u0 + (unit * dv + col) * CHUNK + rb * 16 + (lane & 3) * 2;
#pragma unroll
            for (int j = 0; j < 2; ++j) *(float2*)(to + j * 8) = make_float2(y[j][half * 2], y[j][half * 2 + 1]);
          }
        } else {
          const int at = (rb * 16 + beside + r) * kp + col0 + own;
          stmatrix_x4_trans(smem_u32(wh + at), xh[m][rb]);
          stmatrix_x4_trans(smem_u32(wl + at), xl[m][rb]);
        }
      }
    }
  }
  __syncthreads();
  // W and K leave as they lie.
  const int pieces = 3 * CHUNK * kp / 8;
  uint4* to = (uint4*)(p.wk + unit * 3 * CHUNK * kp);
#pragma unroll 4
  for (int e = tid; e < pieces; e += SOLVE_THREADS) to[e] = ((const uint4*)raw)[e];
}

// ---------------------------------------------------------------------------------------
// chunked: pass
// ---------------------------------------------------------------------------------------
constexpr int PASS_THREADS = 256, PASS_WARPS = PASS_THREADS / 32;
constexpr int PASS_COLUMNS = 16;              // value columns of a block
constexpr int PART_PITCH = CHUNK + 8;         // floats between rows of a partial product
constexpr int U_PITCH = CHUNK + 8;
constexpr size_t SMEM_MOST = 220 * 1024;      // beside some kilobytes of static shared memory

__host__ __device__ inline size_t pass_smem(int n, int stages) {
  return 2 * (size_t)stages * 3 * CHUNK * pitch_of(n) + sizeof(float) * (size_t)PASS_WARPS * PASS_COLUMNS * PART_PITCH;
}

// From chunk to chunk, 16 value columns of a head of a request a block. The state never leaves the registers: a
// warp holds S^T, 16 columns by its own 16 key channels (or twice as many), as the accumulators of the update S^T <-
// exp(c_last) S^T + U^T K, which as they lie are the operand of its share of (W S)^T = S^T W^T. The warps' shares
// are added up through shared memory.
__global__ void __launch_bounds__(PASS_THREADS, 2) delta_pass_kernel(const Delta p, int stages) {
  dependent_launch_prologue();
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ __align__(16) __nv_bfloat16 us[2][PASS_COLUMNS][U_PITCH];      // exp(c_last - c_j) U_j / |k_j| as a sum of two
  __shared__ __align__(16) float weight[CHUNK];                             // exp(c_last - c_j) / |k_j|
  const int d0 = blockIdx.x * PASS_COLUMNS, h = blockIdx.y, i = blockIdx.z, b = p.list != nullptr ? p.list[i] : i;
  const int first = p.q_start[b], count = p.q_start[b + 1] - first;
  if (count <= 1) return;
  const int chunks = (count + CHUNK - 1) / CHUNK;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mid = lane >> 3, r = lane & 7;
  const int n = p.n, dv = p.dv, np = padded(n), kp = np + 8, tiles = np / 16;
  const size_t stage_size = (size_t)3 * CHUNK * kp;
  __nv_bfloat16* ring = (__nv_bfloat16*)raw;                     // per stage W hi, W lo, K: [CHUNK][kp] each
  float* part = (float*)(ring + stages * stage_size);            // [PASS_WARPS][PASS_COLUMNS][PART_PITCH]
  const int parts = min(tiles, PASS_WARPS);
  // A thread adds up, and turns into U, four tokens of one column.
  const int my_col = tid >> 4, my_row = (tid & 15) * 4;
  const bool my_valid = d0 + my_col < dv;
  // What lies in scratch per chunk and head: a chunk on, `heads` units on.
  const size_t unit0 = (size_t)chunk_slot(first, i, 0) * p.heads + h, heads = p.heads;
  const int pieces = 3 * CHUNK * kp / 8, whole = pieces / PASS_THREADS * PASS_THREADS;
  const uint4* wk_at = (const uint4*)(p.wk + unit0 * 3 * CHUNK * kp) + tid;
  const float* vec_at = p.vec + unit0 * 2 * CHUNK;
  const float* u0_at = p.u0 + (unit0 * dv + d0 + my_col) * CHUNK + my_row;
  __nv_bfloat16* u_at = p.u + (unit0 * 2 * dv + d0 + my_col) * CHUNK + my_row;
  __nv_bfloat16* before_at = p.before + (unit0 * 2 * dv + d0 + (lane >> 2)) * n + warp * 16 + (lane & 3) * 2;
  const size_t wk_step = heads * pieces, vec_step = heads * 2 * CHUNK, u0_step = heads * dv * CHUNK, u_step = 2 * u0_step, before_step = heads * 2 * dv * n;
  const size_t lo_state = (size_t)dv * n, lo_u = (size_t)dv * CHUNK;
  const uint32_t ring_at = smem_u32(ring) + tid * 16, ring_other = stages > 1 ? (uint32_t)(stage_size * 2) : 0;
  auto fetch = [&](int chunk) {                                  // W and K of the next chunk, as they lie
    const uint32_t to = ring_at + (chunk & 1 ? ring_other : 0);
#pragma unroll 4
    for (int e = 0; e < whole; e += PASS_THREADS) cp_async16(to + e * 16, wk_at + e);
    if (whole + tid < pieces) cp_async16(to + whole * 16, wk_at + whole);
    cp_async_commit();
    wk_at += wk_step;
  };
  // What a chunk needs in registers, asked for a chunk ahead: U0, c at its end and at token tid, and 1 / |k| there.
  float4 u0 = make_float4(0.f, 0.f, 0.f, 0.f), next_u0 = u0;
  float next_last = 0.f, next_c = 0.f, next_inv = 0.f;
  auto ask = [&]() {
    next_last = vec_at[CHUNK - 1];
    next_c = vec_at[tid & (CHUNK - 1)];
    next_inv = vec_at[CHUNK + (tid & (CHUNK - 1))];
    if (my_valid) next_u0 = *(const float4*)u0_at;
    vec_at += vec_step;
    u0_at += u0_step;
  };
  float* st = p.state + (size_t)p.state_slot[b] * p.slot_stride + (size_t)h * n * dv;
  // s[m][j][e]: column (lane >> 2) + (e >> 1) 8, key channel (warp + 8 m) 16 + j 8 + (lane & 3) 2 + (e & 1)
  float s[2][2][4];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = (warp + 8 * m) * 16 + j * 8 + (lane & 3) * 2 + (e & 1), col = d0 + (lane >> 2) + (e >> 1) * 8;
        s[m][j][e] = key < n && col < dv ? st[(size_t)key * dv + col] : 0.f;
      }
  fetch(0);
  ask();
  for (int chunk = 0; chunk < chunks; ++chunk) {
    cp_async_wait<0>();
    __syncthreads();                     // this chunk's W and K are there; the chunk before is done with
    if (stages > 1 && chunk + 1 < chunks) fetch(chunk + 1);
    const float last = next_last, keep = exp2f(last);
    u0 = next_u0;
    if (tid < CHUNK) weight[tid] = exp2f(last - next_c) * next_inv;
    if (chunk + 1 < chunks) ask();
    const __nv_bfloat16* wh = ring + (stages > 1 ? chunk & 1 : 0) * stage_size;
    const __nv_bfloat16* ks = wh + (size_t)2 * CHUNK * kp;
    float acc[CHUNK / 8][4];
#pragma unroll
    for (int j = 0; j < CHUNK / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const int key0 = (warp + 8 * m) * 16;
      if (key0 >= np) break;
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) split_pair(s[m][e >> 1][(e & 1) * 2], s[m][e >> 1][(e & 1) * 2 + 1], hi[e], lo[e]);
      const uint32_t w_at = smem_u32(wh + (size_t)((mid >> 1) * 8 + r) * kp + key0 + (mid & 1) * 8), w_lo = CHUNK * kp * 2;
      // the three products of an accumulator stand eight others apart: none waits for the one before it
      uint32_t w4[CHUNK / 16][4];
#pragma unroll
      for (int j = 0; j < CHUNK / 16; ++j) ldmatrix_x4(w4[j], w_at + j * 16 * kp * 2);
#pragma unroll
      for (int j = 0; j < CHUNK / 8; ++j) mma_16816(acc[j], hi, w4[j >> 1][2 * (j & 1)], w4[j >> 1][2 * (j & 1) + 1]);
#pragma unroll
      for (int j = 0; j < CHUNK / 8; ++j) mma_16816(acc[j], lo, w4[j >> 1][2 * (j & 1)], w4[j >> 1][2 * (j & 1) + 1]);
#pragma unroll
      for (int j = 0; j < CHUNK / 16; ++j) ldmatrix_x4(w4[j], w_at + j * 16 * kp * 2 + w_lo);
#pragma unroll
      for (int j = 0; j < CHUNK / 8; ++j) mma_16816(acc[j], hi, w4[j >> 1][2 * (j & 1)], w4[j >> 1][2 * (j & 1) + 1]);
      // the state before this chunk goes to the output kernel
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (key0 + (e >> 1) * 8 + (lane & 3) * 2 < n && d0 + (lane >> 2) + (e & 1) * 8 < dv) {
          __nv_bfloat16* to = before_at + m * 128 + (e >> 1) * 8 + (e & 1) * 8 * n;
          *(uint32_t*)to = hi[e];
          *(uint32_t*)(to + lo_state) = lo[e];
        }
      }
    }
    before_at += before_step;
    if (warp < parts) {
      float* to = part + ((size_t)warp * PASS_COLUMNS + (lane >> 2)) * PART_PITCH + (lane & 3) * 2;
#pragma unroll
      for (int j = 0; j < CHUNK / 8; ++j) {
        *(float2*)(to + j * 8) = make_float2(acc[j][0], acc[j][1]);
        *(float2*)(to + 8 * PART_PITCH + j * 8) = make_float2(acc[j][2], acc[j][3]);
      }
    }
    __syncthreads();
    {
      float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
      const float* from = part + (size_t)my_col * PART_PITCH + my_row;
#pragma unroll
      for (int w = 0; w < PASS_WARPS; ++w) {
        if (w >= parts) break;
        const float4 x = *(const float4*)(from + (size_t)w * PASS_COLUMNS * PART_PITCH);
        sum.x += x.x, sum.y += x.y, sum.z += x.z, sum.w += x.w;
      }
      const float4 f = *(const float4*)(weight + my_row);
      const float u[4] = {u0.x - sum.x, u0.y - sum.y, u0.z - sum.z, u0.w - sum.w};
      uint2 hi, lo;
      split_pair(u[0] * f.x, u[1] * f.y, hi.x, lo.x);
      split_pair(u[2] * f.z, u[3] * f.w, hi.y, lo.y);
      *(uint2*)&us[0][my_col][my_row] = hi;
      *(uint2*)&us[1][my_col][my_row] = lo;
      if (my_valid) {
        split_pair(u[0], u[1], hi.x, lo.x);
        split_pair(u[2], u[3], hi.y, lo.y);
        *(uint2*)u_at = hi;
        *(uint2*)(u_at + lo_u) = lo;
      }
      u_at += u_step;
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const int key0 = (warp + 8 * m) * 16;
      if (key0 >= np) break;
      float more[2][4];                  // the low halves' products, a chain of their own
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[m][j][e] *= keep, more[j][e] = 0.f;
#pragma unroll
      for (int t = 0; t < CHUNK / 16; ++t) {
        uint32_t hi[4], lo[4], k4[4];
        ldmatrix_x4(hi, smem_u32(&us[0][(mid & 1) * 8 + r][t * 16 + (mid >> 1) * 8]));
        ldmatrix_x4(lo, smem_u32(&us[1][(mid & 1) * 8 + r][t * 16 + (mid >> 1) * 8]));
        ldmatrix_x4_trans(k4, smem_u32(ks + (size_t)(t * 16 + (mid & 1) * 8 + r) * kp + key0 + (mid >> 1) * 8));
#pragma unroll
        for (int j = 0; j < 2; ++j) mma_16816(s[m][j], hi, k4[2 * j], k4[2 * j + 1]);
#pragma unroll
        for (int j = 0; j < 2; ++j) mma_16816(more[j], lo, k4[2 * j], k4[2 * j + 1]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[m][j][e] += more[j][e];
    }
    if (stages == 1 && chunk + 1 < chunks) {
      __syncthreads();                   // K is used up
      fetch(chunk + 1);
    }
  }
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = (warp + 8 * m) * 16 + j * 8 + (lane & 3) * 2 + (e & 1), col = d0 + (lane >> 2) + (e >> 1) * 8;
        if (key < n && col < dv) st[(size_t)key * dv + col] = s[m][j][e];
      }
}

// ---------------------------------------------------------------------------------------
// chunked: output
// ---------------------------------------------------------------------------------------
constexpr int OUT_THREADS = 256, OUT_DVT = 64;
__host__ __device__ inline size_t output_smem(int n) {
  const int np = (n + 15) & ~15;
  return 2 * ((size_t)2 * (CHUNK + OUT_DVT) * (np + 8) + (size_t)2 * OUT_DVT * U_PITCH);
}

// A chunk's read-outs, 64 value columns a block: a warp 16 tokens x 32 columns.
__global__ void __launch_bounds__(OUT_THREADS) delta_output_kernel(const Delta p) {
  dependent_launch_prologue();
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ __align__(16) float cumulative[CHUNK], k_inv[CHUNK], q_inv[CHUNK];
  const int dv_tiles = (p.dv + OUT_DVT - 1) / OUT_DVT;
  const int d0 = (blockIdx.x % dv_tiles) * OUT_DVT, chunk = blockIdx.x / dv_tiles;
  const int h = blockIdx.y, i = blockIdx.z, b = p.list != nullptr ? p.list[i] : i;
  const int first = p.q_start[b], all = p.q_start[b + 1] - first;
  const int count = min(CHUNK, all - chunk * CHUNK);
  if (all == 1 || count <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mid = lane >> 3, r = lane & 7;
  const int n = p.n, dv = p.dv, np = (n + 15) & ~15, kp = np + 8, g = h / (p.heads / p.groups);
  const size_t token0 = (size_t)first + chunk * CHUNK;
  const size_t unit = (size_t)chunk_slot(first, i, chunk) * p.heads + h;
  __nv_bfloat16* qs = (__nv_bfloat16*)raw;                // [CHUNK][kp]
  __nv_bfloat16* ks = qs + (size_t)CHUNK * kp;
  __nv_bfloat16* sh = ks + (size_t)CHUNK * kp;            // [OUT_DVT][kp]
  __nv_bfloat16* sl = sh + (size_t)OUT_DVT * kp;
  __nv_bfloat16* uh = sl + (size_t)OUT_DVT * kp;          // [OUT_DVT][U_PITCH]
  __nv_bfloat16* ul = uh + (size_t)OUT_DVT * U_PITCH;
  const int valid = min(OUT_DVT, dv - d0);
  fetch_rows(qs, kp, (const __nv_bfloat16*)p.q + token0 * p.q_ld + g * n, p.q_ld, CHUNK, count, np, n);
  fetch_rows(ks, kp, (const __nv_bfloat16*)p.k + token0 * p.k_ld + g * n, p.k_ld, CHUNK, count, np, n);
  const __nv_bfloat16* before = p.before + (unit * 2 * dv + d0) * n;
  fetch_rows(sh, kp, before, n, OUT_DVT, valid, np, n);
  fetch_rows(sl, kp, before + (size_t)dv * n, n, OUT_DVT, valid, np, n);
  cp_async_commit();
  const __nv_bfloat16* u = p.u + (unit * 2 * dv + d0) * CHUNK;
  fetch_rows(uh, U_PITCH, u, CHUNK, OUT_DVT, valid, CHUNK, CHUNK);
  fetch_rows(ul, U_PITCH, u + (size_t)dv * CHUNK, CHUNK, OUT_DVT, valid, CHUNK, CHUNK);
  cp_async_commit();
  if (tid < CHUNK) {
    cumulative[tid] = p.vec[unit * 2 * CHUNK + tid];
    k_inv[tid] = p.vec[unit * 2 * CHUNK + CHUNK + tid];
  }
  cp_async_wait<1>();
  __syncthreads();
  {
    const float qq = row_squares(qs, kp, np, tid >> 2);
    if ((tid & 3) == 0) q_inv[tid >> 2] = inverse_root(qq + p.key_eps) * p.q_scale;
  }
  const int tile = warp & 3, row0 = tile * 16, col0 = (warp >> 2) * 32;
  float acc[4][4];
#pragma unroll
  for (int j = 0; j < 4; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
  const uint32_t q_at = smem_u32(qs + (size_t)(row0 + (mid & 1) * 8 + r) * kp + (mid >> 1) * 8);
#pragma unroll 2
  for (int t = 0; t < np / 16; ++t) {
    uint32_t a[4];
    ldmatrix_x4(a, q_at + t * 32);
#pragma unroll
    for (int plane = 0; plane < 2; ++plane) {
      const __nv_bfloat16* from = (plane == 0 ? sh : sl) + (size_t)(col0 + (mid >> 1) * 8 + r) * kp + t * 16 + (mid & 1) * 8;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        uint32_t s4[4];
        ldmatrix_x4(s4, smem_u32(from + (size_t)j * 16 * kp));
        mma_16816(acc[2 * j], a, s4[0], s4[1]);
        mma_16816(acc[2 * j + 1], a, s4[2], s4[3]);
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  const int rows[2] = {row0 + (lane >> 2), row0 + (lane >> 2) + 8};
  const float at_row[2] = {cumulative[rows[0]], cumulative[rows[1]]}, scale[2] = {q_inv[rows[0]], q_inv[rows[1]]};
  const float from_before[2] = {exp2f(at_row[0]) * scale[0], exp2f(at_row[1]) * scale[1]};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    acc[j][0] *= from_before[0];
    acc[j][1] *= from_before[0];
    acc[j][2] *= from_before[1];
    acc[j][3] *= from_before[1];
  }
  for (int t = 0; t <= tile; ++t) {                      // 16 earlier tokens at a time
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    const uint32_t k_at = smem_u32(ks + (size_t)(t * 16 + (mid >> 1) * 8 + r) * kp + (mid & 1) * 8);
#pragma unroll 4
    for (int x = 0; x < np / 16; ++x) {
      uint32_t a[4], k4[4];
      ldmatrix_x4(a, q_at + x * 32);
      ldmatrix_x4(k4, k_at + x * 32);
      mma_16816(s[0], a, k4[0], k4[1]);
      mma_16816(s[1], a, k4[2], k4[3]);
    }
#pragma unroll
    for (int w = 0; w < 2; ++w) {
      const int token = t * 16 + w * 8 + (lane & 3) * 2;
      const float2 c2 = *(const float2*)(cumulative + token), i2 = *(const float2*)(k_inv + token);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int half = e >> 1;
        const float f = scale[half] * (e & 1 ? i2.y : i2.x) * fast_exp2(at_row[half] - (e & 1 ? c2.y : c2.x));
        s[w][e] = token + (e & 1) <= rows[half] ? s[w][e] * f : 0.f;
      }
    }
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) split_pair(s[e >> 1][(e & 1) * 2], s[e >> 1][(e & 1) * 2 + 1], hi[e], lo[e]);
    uint32_t u4[2][4], l4[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int at = (col0 + j * 16 + (mid >> 1) * 8 + r) * U_PITCH + t * 16 + (mid & 1) * 8;
      ldmatrix_x4(u4[j], smem_u32(uh + at));
      ldmatrix_x4(l4[j], smem_u32(ul + at));
    }
#pragma unroll
    for (int x = 0; x < 3; ++x)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const uint32_t* from = x == 2 ? l4[j >> 1] : u4[j >> 1];
        mma_16816(acc[j], x == 1 ? lo : hi, from[2 * (j & 1)], from[2 * (j & 1) + 1]);
      }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    if (rows[e] >= count) continue;
    float* out = p.o + ((token0 + rows[e]) * p.heads + h) * dv + d0;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = col0 + j * 8 + (lane & 3) * 2;
      if (d0 + col < dv) *(float2*)(out + col) = make_float2(acc[j][e * 2], acc[j][e * 2 + 1]);
    }
  }
}

int check_delta(const Delta& p, int entries) {
  if (p.heads < 1 || p.groups < 1 || p.heads % p.groups) return fail(2, "gated_delta: %d heads in %d groups", p.heads, p.groups);
  if (p.n < 1 || p.dv < 1 || p.n > 1024) return fail(2, "gated_delta: heads of %d key and %d value channels", p.n, p.dv);
  if (p.heads > 65535 || entries > 65535) return fail(3, "gated_delta: %d heads x %d requests exceed one launch", p.heads, entries);
  return 0;
}

Delta delta_of(float* o, float* state, long long slot_stride, const void* q, int q_ld, const void* k, int k_ld, const void* v, int v_ld,
               const float* log_decay, const float* beta, float key_eps, float q_scale, const int* q_start, const int* state_slot, int heads,
               int groups, int n, int dv) {
  Delta p{};
  p.q = q, p.k = k, p.v = v;
  p.log_decay = log_decay, p.beta = beta;
  p.o = o, p.state = state;
  p.q_start = q_start, p.state_slot = state_slot;
  p.slot_stride = slot_stride;
  p.q_ld = q_ld, p.k_ld = k_ld, p.v_ld = v_ld;
  p.heads = heads, p.groups = groups, p.n = n, p.dv = dv;
  p.key_eps = key_eps, p.q_scale = q_scale;
  return p;
}

int launch_pass(const Delta& p, int listed, cudaStream_t s) {
  // Two stages of W and K while every block has an SM to itself; one when there are more blocks, which then share SMs.
  const dim3 grid((p.dv + PASS_COLUMNS - 1) / PASS_COLUMNS, p.heads, listed);
  const bool alone = (long long)grid.x * grid.y * grid.z <= 148;
  const int stages = alone && pass_smem(p.n, 2) <= SMEM_MOST ? 2 : 1;
  if (int err = allow_smem(delta_pass_kernel, SMEM_MOST, "gated_delta_chunked")) return err;
  launch_kernel(delta_pass_kernel, grid, PASS_THREADS, pass_smem(p.n, stages), s, p, stages);
  return check_launch("gated_delta_pass");
}

}  // namespace

// Token after token. skip_single: the entries of one token are left to `pae_gated_delta_step`.
PAE_EXPORT int pae_gated_delta_scan(float* o, float* state, long long slot_stride, const void* q, int q_ld, const void* k, int k_ld,
                                    const void* v, int v_ld, const float* log_decay, const float* beta, float key_eps, float q_scale,
                                    const int* q_start, const int* state_slot, int entries, int heads, int groups, int n, int dv,
                                    int skip_single, int dtype, void* stream) {
  if (entries == 0) return 0;
  Delta p = delta_of(o, state, slot_stride, q, q_ld, k, k_ld, v, v_ld, log_decay, beta, key_eps, q_scale, q_start, state_slot, heads, groups, n, dv);
  p.skip_single = skip_single;
  if (int err = check_delta(p, entries)) return err;
  if (dtype == kF32) return scan_of<float>(p, entries, (cudaStream_t)stream);
  if (dtype == kBF16) return scan_of<__nv_bfloat16>(p, entries, (cudaStream_t)stream);
  return fail(1, "gated_delta_scan: unknown dtype %d", dtype);
}

// 1 when the step kernel takes these sizes (16-byte pieces of the state).
PAE_EXPORT int pae_gated_delta_step_supports(int n, int dv, long long slot_stride) {
  return n >= 1 && n <= 1024 && dv % 4 == 0 && slot_stride % 4 == 0 ? 1 : 0;
}

// The entries that bring one token.
PAE_EXPORT int pae_gated_delta_step(float* o, float* state, long long slot_stride, const void* q, int q_ld, const void* k, int k_ld,
                                    const void* v, int v_ld, const float* log_decay, const float* beta, float key_eps, float q_scale,
                                    const int* q_start, const int* state_slot, int entries, int heads, int groups, int n, int dv,
                                    int dtype, void* stream) {
  if (entries == 0) return 0;
  const Delta p = delta_of(o, state, slot_stride, q, q_ld, k, k_ld, v, v_ld, log_decay, beta, key_eps, q_scale, q_start, state_slot, heads, groups, n, dv);
  if (int err = check_delta(p, entries)) return err;
  if (!pae_gated_delta_step_supports(n, dv, slot_stride) || (((uintptr_t)state | (uintptr_t)o) & 15))
    return fail(2, "gated_delta_step: a state of %d x %d is not made of aligned 16-byte pieces", n, dv);
  if (dtype == kF32) return step_of<float>(p, entries, (cudaStream_t)stream);
  if (dtype == kBF16) return step_of<__nv_bfloat16>(p, entries, (cudaStream_t)stream);
  return fail(1, "gated_delta_step: unknown dtype %d", dtype);
}

// 1 when the chunked kernels take these sizes: rows of 16-byte pieces, up to 256 key channels.
PAE_EXPORT int pae_gated_delta_chunked_supports(int n, int dv, int q_ld, int k_ld, int v_ld, long long slot_stride) {
  return n % 8 == 0 && dv % 8 == 0 && n <= 256 && solve_smem(n, dv) <= SMEM_MOST && q_ld % 8 == 0 && k_ld % 8 == 0 && v_ld % 8 == 0 && slot_stride % 2 == 0 ? 1 : 0;
}

PAE_EXPORT int pae_gated_delta_chunk() { return CHUNK; }
PAE_EXPORT int pae_gated_delta_pitch(int n) { return pitch_of(n); }

// The entries that bring more than one token, bfloat16. list: `listed` entries to look at (null: all, and
// those of one token are passed over). Scratch for tokens / 64 + listed chunks, per chunk and head: wk bfloat16
// [3, 64, pitch], u0 floats [dv, 64], u bfloat16 [2, dv, 64], before bfloat16 [2, dv, n], vec floats [2, 64]. Three launches.
PAE_EXPORT int pae_gated_delta_chunked(float* o, float* state, long long slot_stride, const void* q, int q_ld, const void* k, int k_ld,
                                       const void* v, int v_ld, const float* log_decay, const float* beta, float key_eps, float q_scale,
                                       const int* q_start, const int* state_slot, const int* list, int listed, int max_q_len, int heads,
                                       int groups, int n, int dv, void* wk, float* u0, void* u, void* before, float* vec, void* stream) {
  if (listed == 0 || max_q_len <= 1) return 0;
  Delta p = delta_of(o, state, slot_stride, q, q_ld, k, k_ld, v, v_ld, log_decay, beta, key_eps, q_scale, q_start, state_slot, heads, groups, n, dv);
  p.list = list;
  p.wk = (__nv_bfloat16*)wk, p.u0 = u0, p.u = (__nv_bfloat16*)u, p.before = (__nv_bfloat16*)before, p.vec = vec;
  if (int err = check_delta(p, listed)) return err;
  if (!pae_gated_delta_chunked_supports(n, dv, q_ld, k_ld, v_ld, slot_stride))
    return fail(2, "gated_delta_chunked: heads of %d key and %d value channels", n, dv);
  if (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state | (uintptr_t)wk | (uintptr_t)u0 | (uintptr_t)u | (uintptr_t)before) & 15)
    return fail(2, "gated_delta_chunked: an operand does not start on a 16-byte boundary");
  cudaStream_t s = (cudaStream_t)stream;
  const int chunks = (max_q_len + CHUNK - 1) / CHUNK;
  if (int err = allow_smem(delta_solve_kernel, SMEM_MOST, "gated_delta_chunked")) return err;
  launch_kernel(delta_solve_kernel, dim3(chunks, heads, listed), SOLVE_THREADS, solve_smem(n, dv), s, p);
  if (int err = check_launch("gated_delta_solve")) return err;
  if (int err = launch_pass(p, listed, s)) return err;
  if (int err = allow_smem(delta_output_kernel, SMEM_MOST, "gated_delta_chunked")) return err;
  launch_kernel(delta_output_kernel, dim3(chunks * ((dv + OUT_DVT - 1) / OUT_DVT), heads, listed), OUT_THREADS, output_smem(n), s, p);
  return check_launch("gated_delta_output");
}

PAE_DEFINE_LAST_ERROR()

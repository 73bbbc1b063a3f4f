// What stands around the recurrence of a selective state space (Mamba-2) and of other gated linear
// mixers (the recurrence itself is in decay_memory.cu).
//
// `ssm_prepare`, from the fused input projection z | x B C | dt, float32 (or the planes of a split
// product, added here in their order), per token:
//   u_c = silu(bias_c + sum_j taps[c, j] raw[t - taps + 1 + j, c])      every channel of x, B and C
//   step_h = softplus(dt_h + dt_bias_h)          log_decay_h = -exp(A_log_h) step_h
//   beta_h = sigmoid(b_h)                        for a mixer that has such columns (the gated delta rule)
// The last taps - 1 raw rows of a request are kept as per-request state, so a portion's first tokens
// read the rows before it; zeros stand before a sequence's start. The thread that owns a channel of
// a portion's first tokens reads the old rows, uses them, and puts the portion's last rows in
// their place: no other thread reads them. All arithmetic is float32; u leaves in the engine's
// element type, step and log_decay in float32.
//
// `gated_group_norm`: the channels of a token in equal groups, each divided by its own root mean
// square, with a gate silu(g) per channel before or after the division:
//   gate first   out = rms(y * silu(g)) * weight        gate last   out = rms(y) * weight * silu(g)
// times a constant, into a column range of the output's rows.
#include "common.cuh"

using namespace pae;

namespace {

constexpr int TOKENS = 16;            // of a block, and at least taps - 1
constexpr int THREADS = 128;

struct Prepare {
  const float* proj;        // [planes, tokens, ld]
  const float* taps_w;      // [channels, taps]
  const float* bias;        // [channels] or null
  const float* dt_bias;     // [heads]
  const float* a_log;       // [heads]
  float* state;             // slot s: state + s * slot_stride, [taps - 1, channels]
  void* u;                  // [tokens, channels]
  float* step;              // [tokens, heads]
  float* log_decay;         // [tokens, heads]
  float* beta;              // [tokens, heads] or null
  float* z;                 // [tokens, z_cols]: the gate's columns, summed; null: they stay in proj
  const int* q_start;
  const int* q_pos0;
  const int* state_slot;
  long long slot_stride, plane;
  int planes, ld, z_off, z_cols, u_off, channels, dt_off, beta_off, heads, taps;
  int u_blocks, z_blocks;   // blockIdx.x: channels of u, then of z, then heads of the block's tokens
};

template <int VEC>
struct Values {
  float x[VEC];
};

template <int VEC>
__device__ __forceinline__ Values<VEC> load(const float* from) {
  Values<VEC> v;
  if (VEC == 4) {
    const float4 f = *(const float4*)from;
    v.x[0] = f.x, v.x[1 % VEC] = f.y, v.x[2 % VEC] = f.z, v.x[3 % VEC] = f.w;
  } else {
    v.x[0] = *from;
  }
  return v;
}

template <int VEC>
__device__ __forceinline__ void store(float* to, const Values<VEC>& v) {
  if (VEC == 4)
    *(float4*)to = make_float4(v.x[0], v.x[1 % VEC], v.x[2 % VEC], v.x[3 % VEC]);
  else
    *to = v.x[0];
}

template <int VEC>
__device__ __forceinline__ void store(__nv_bfloat16* to, const Values<VEC>& v) {
  if (VEC == 4) {
    uint2 packed;
    *(__nv_bfloat162*)&packed.x = __floats2bfloat162_rn(v.x[0], v.x[1 % VEC]);
    *(__nv_bfloat162*)&packed.y = __floats2bfloat162_rn(v.x[2 % VEC], v.x[3 % VEC]);
    *(uint2*)to = packed;
  } else {
    *to = __float2bfloat16_rn(v.x[0]);
  }
}

// silu whose result leaves as T: for bfloat16 by the hardware's exponential and reciprocal (some units of
// 2^-22 off, far below the rounding that follows).
template <typename T>
__device__ __forceinline__ float silu(float x) {
  return x / (1.f + expf(-x));
}
template <>
__device__ __forceinline__ float silu<__nv_bfloat16>(float x) {
  return __fdividef(x, 1.f + __expf(-x));
}

// A value of the projection, its planes added up.
template <int VEC>
__device__ __forceinline__ Values<VEC> projected(const Prepare& p, size_t token, int col) {
  const float* from = p.proj + token * p.ld + col;
  Values<VEC> v = load<VEC>(from);
  for (int k = 1; k < p.planes; ++k) {
    const Values<VEC> more = load<VEC>(from + (size_t)k * p.plane);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v.x[j] += more.x[j];
  }
  return v;
}

// TAPS > 0: known when compiled, the window of rows stays in registers; 0: any number up to TOKENS + 1.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(THREADS) ssm_prepare_kernel(const Prepare p) {
  dependent_launch_prologue();
  const int b = blockIdx.z, t0 = blockIdx.y * TOKENS;
  const int first = p.q_start[b], count = p.q_start[b + 1] - first;
  const int tokens = min(TOKENS, count - t0);
  if (tokens <= 0) return;
  int x_block = blockIdx.x;
  if (x_block >= p.u_blocks) {
    x_block -= p.u_blocks;
    if (x_block < p.z_blocks) {
      const int c = (x_block * THREADS + threadIdx.x) * VEC;
      if (c >= p.z_cols) return;
      for (int t = 0; t < tokens; ++t) {
        const size_t token = (size_t)first + t0 + t;
        store<VEC>(p.z + token * p.z_cols + c, projected<VEC>(p, token, p.z_off + c));
      }
      return;
    }
    const int e = (x_block - p.z_blocks) * THREADS + threadIdx.x;       // a head of a token
    if (e >= tokens * p.heads) return;
    const int t = e / p.heads, h = e - t * p.heads;
    const size_t token = (size_t)first + t0 + t;
    const float x = projected<1>(p, token, p.dt_off + h).x[0] + p.dt_bias[h];
    const float step = fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
    p.step[token * p.heads + h] = step;
    p.log_decay[token * p.heads + h] = -expf(p.a_log[h]) * step;
    if (p.beta != nullptr) p.beta[token * p.heads + h] = 1.f / (1.f + expf(-projected<1>(p, token, p.beta_off + h).x[0]));
    return;
  }
  const int c = (x_block * THREADS + threadIdx.x) * VEC;
  if (c >= p.channels) return;
  const int taps = TAPS > 0 ? TAPS : p.taps, kept = taps - 1;
  const int pos0 = p.q_pos0[b];
  float* mine = p.state + (size_t)p.state_slot[b] * p.slot_stride + c;
  auto raw = [&](int rel) -> Values<VEC> {             // the row `rel` tokens after the portion's first
    if (rel >= 0) return projected<VEC>(p, (size_t)first + rel, p.u_off + c);
    Values<VEC> none;
#pragma unroll
    for (int j = 0; j < VEC; ++j) none.x[j] = 0.f;
    return pos0 + rel < 0 ? none : load<VEC>(mine + (size_t)(kept + rel) * p.channels);
  };
  Values<VEC> bias;
#pragma unroll
  for (int j = 0; j < VEC; ++j) bias.x[j] = p.bias != nullptr ? p.bias[c + j] : 0.f;
  T* out = (T*)p.u + ((size_t)first + t0) * p.channels + c;
  if (TAPS > 0) {
    constexpr int N = TAPS > 0 ? TAPS : 1;
    Values<VEC> window[N];
    float w[N][VEC];
#pragma unroll
    for (int j = 0; j < N; ++j)
#pragma unroll
      for (int v = 0; v < VEC; ++v) w[j][v] = p.taps_w[(size_t)(c + v) * N + j];
#pragma unroll
    for (int j = 0; j + 1 < N; ++j) window[j + 1] = raw(t0 - (N - 1) + j);
    constexpr int AHEAD = 8;              // rows asked for at a time
    for (int t1 = 0; t1 < tokens; t1 += AHEAD) {
      Values<VEC> rows[AHEAD];
#pragma unroll
      for (int i = 0; i < AHEAD; ++i)
        if (t1 + i < tokens) rows[i] = projected<VEC>(p, (size_t)first + t0 + t1 + i, p.u_off + c);
#pragma unroll
      for (int i = 0; i < AHEAD; ++i) {
        if (t1 + i >= tokens) break;
#pragma unroll
        for (int j = 0; j + 1 < N; ++j) window[j] = window[j + 1];
        window[N - 1] = rows[i];
        Values<VEC> acc = bias;
#pragma unroll
        for (int j = 0; j < N; ++j)
#pragma unroll
          for (int v = 0; v < VEC; ++v) acc.x[v] = fmaf(w[j][v], window[j].x[v], acc.x[v]);
#pragma unroll
        for (int v = 0; v < VEC; ++v) acc.x[v] = silu<T>(acc.x[v]);
        store<VEC>(out + (size_t)(t1 + i) * p.channels, acc);
      }
    }
  } else {
    for (int t = 0; t < tokens; ++t) {
      Values<VEC> acc = bias;
      for (int j = 0; j < taps; ++j) {
        const Values<VEC> u = raw(t0 + t - kept + j);
#pragma unroll
        for (int v = 0; v < VEC; ++v) acc.x[v] = fmaf(p.taps_w[(size_t)(c + v) * taps + j], u.x[v], acc.x[v]);
      }
#pragma unroll
      for (int v = 0; v < VEC; ++v) acc.x[v] = silu<T>(acc.x[v]);
      store<VEC>(out + (size_t)t * p.channels, acc);
    }
  }
  // Row i of the state becomes the row that stands kept - i before the next portion; walking i upwards,
  // an old row is read before its place is written.
  if (t0 == 0)
    for (int i = 0; i < kept; ++i) store<VEC>(mine + (size_t)i * p.channels, raw(count - kept + i));
}

template <typename T, int VEC>
void launch_prepare(const Prepare& p, dim3 grid, cudaStream_t s) {
  switch (p.taps) {
    case 1: launch_kernel(ssm_prepare_kernel<T, VEC, 1>, grid, THREADS, 0, s, p); break;
    case 2: launch_kernel(ssm_prepare_kernel<T, VEC, 2>, grid, THREADS, 0, s, p); break;
    case 3: launch_kernel(ssm_prepare_kernel<T, VEC, 3>, grid, THREADS, 0, s, p); break;
    case 4: launch_kernel(ssm_prepare_kernel<T, VEC, 4>, grid, THREADS, 0, s, p); break;
    default: launch_kernel(ssm_prepare_kernel<T, VEC, 0>, grid, THREADS, 0, s, p); break;
  }
}

struct GroupNorm {
  const float* y;           // [tokens, width]
  const float* gate;        // [tokens, gate_ld], columns from gate_off
  const float* weight;      // [width] or null
  void* out;                // [tokens, out_ld], columns from out_off
  int groups, size, gate_ld, gate_off, out_ld, out_off, gate_first;
  float eps, mult;
};

// A group belongs to one warp (WIDE false: four groups a block) or to one block.
template <typename T, int VEC, bool WIDE>
__global__ void __launch_bounds__(WIDE ? 256 : 128) gated_group_norm_kernel(const GroupNorm p) {
  dependent_launch_prologue();
  constexpr int LANES = WIDE ? 256 : 32;
  __shared__ float partial[8];
  const int lane = WIDE ? threadIdx.x : threadIdx.x & 31;
  const int group = WIDE ? blockIdx.y : blockIdx.y * 4 + (threadIdx.x >> 5);
  if (group >= p.groups) return;
  const size_t token = blockIdx.x;
  const int c0 = group * p.size;
  const float* y = p.y + token * p.groups * p.size + c0;
  const float* gate = p.gate + token * p.gate_ld + p.gate_off + c0;
  float squares = 0.f;
  // the first KEPT pieces of a thread stay in registers, gated, all of them asked for at once
  constexpr int KEPT = 8;
  Values<VEC> ys[KEPT], gs[KEPT];
#pragma unroll
  for (int k = 0; k < KEPT; ++k) {
    const int i = (lane + k * LANES) * VEC;
    if (i < p.size) ys[k] = load<VEC>(y + i), gs[k] = load<VEC>(gate + i);
  }
#pragma unroll
  for (int k = 0; k < KEPT; ++k) {
    if ((lane + k * LANES) * VEC >= p.size) break;
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const float gated = ys[k].x[j] * silu<T>(gs[k].x[j]), v = p.gate_first ? gated : ys[k].x[j];
      squares = fmaf(v, v, squares);
      ys[k].x[j] = gated;
    }
  }
  for (int i = (lane + KEPT * LANES) * VEC; i < p.size; i += LANES * VEC) {
    Values<VEC> v = load<VEC>(y + i);
    if (p.gate_first) {
      const Values<VEC> g = load<VEC>(gate + i);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v.x[j] *= silu<T>(g.x[j]);
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) squares = fmaf(v.x[j], v.x[j], squares);
  }
  squares = warp_sum(squares);
  if (WIDE) {
    if ((threadIdx.x & 31) == 0) partial[threadIdx.x >> 5] = squares;
    __syncthreads();
    squares = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) squares += partial[w];
  }
  const float scale = p.mult / sqrtf(squares / (float)p.size + p.eps);
  T* out = (T*)p.out + token * p.out_ld + p.out_off + c0;
#pragma unroll
  for (int k = 0; k < KEPT; ++k) {
    const int i = (lane + k * LANES) * VEC;
    if (i >= p.size) break;
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      ys[k].x[j] *= scale;
      if (p.weight != nullptr) ys[k].x[j] *= p.weight[c0 + i + j];
    }
    store<VEC>(out + i, ys[k]);
  }
  for (int i = (lane + KEPT * LANES) * VEC; i < p.size; i += LANES * VEC) {
    Values<VEC> v = load<VEC>(y + i);
    const Values<VEC> g = load<VEC>(gate + i);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      v.x[j] = v.x[j] * silu<T>(g.x[j]) * scale;
      if (p.weight != nullptr) v.x[j] *= p.weight[c0 + i + j];
    }
    store<VEC>(out + i, v);
  }
}

template <typename T, int VEC>
void launch_group_norm(const GroupNorm& p, int tokens, cudaStream_t s) {
  if (p.size > 1024)
    launch_kernel(gated_group_norm_kernel<T, VEC, true>, dim3(tokens, p.groups), 256, 0, s, p);
  else
    launch_kernel(gated_group_norm_kernel<T, VEC, false>, dim3(tokens, (p.groups + 3) / 4), 128, 0, s, p);
}

bool aligned16(const void* ptr) { return (((uintptr_t)ptr) & 15) == 0; }

}  // namespace

// proj float32 [planes][tokens, ld] with z (z_cols columns), u (channels) and dt (heads) at the given
// offsets; u [tokens, channels] in `dtype`; step and log_decay float32 [tokens, heads]; beta likewise or null; z float32 [tokens,
// z_cols] or null. state: slot s holds [taps - 1, channels] floats at state + s * slot_stride.
PAE_EXPORT int pae_ssm_prepare(void* u, float* step, float* log_decay, float* beta, int beta_off, float* z, float* state, long long slot_stride, const float* proj,
                               int planes, int ld, int z_off, int z_cols, int u_off, int channels, int dt_off, int heads,
                               const float* taps_w, int taps, const float* bias, const float* dt_bias, const float* a_log,
                               const int* q_start, const int* q_pos0, const int* state_slot, int tokens, int entries, int max_q_len,
                               int dtype, void* stream) {
  if (tokens == 0 || entries == 0) return 0;
  if (taps < 1 || taps > TOKENS + 1) return fail(2, "ssm_prepare: a convolution of %d taps (1 to %d)", taps, TOKENS + 1);
  if (planes < 1 || channels < 1 || heads < 1) return fail(2, "ssm_prepare: %d planes, %d channels, %d heads", planes, channels, heads);
  if (entries > 65535 || (max_q_len + TOKENS - 1) / TOKENS > 65535)
    return fail(3, "ssm_prepare: %d requests of up to %d tokens exceed one launch", entries, max_q_len);
  Prepare p{};
  p.proj = proj, p.taps_w = taps_w, p.bias = bias, p.dt_bias = dt_bias, p.a_log = a_log;
  p.state = state, p.u = u, p.step = step, p.log_decay = log_decay, p.z = z, p.beta = beta, p.beta_off = beta_off;
  p.q_start = q_start, p.q_pos0 = q_pos0, p.state_slot = state_slot;
  p.slot_stride = slot_stride, p.plane = (long long)tokens * ld;
  p.planes = planes, p.ld = ld, p.z_off = z_off, p.z_cols = z_cols, p.u_off = u_off, p.channels = channels;
  p.dt_off = dt_off, p.heads = heads, p.taps = taps;
  const bool wide = ((ld | z_off | z_cols | u_off | channels) & 3) == 0 && slot_stride % 4 == 0 && p.plane % 4 == 0 && aligned16(proj) &&
                    aligned16(u) && aligned16(state) && (z == nullptr || aligned16(z));
  const int vec = wide ? 4 : 1;
  p.u_blocks = (channels + THREADS * vec - 1) / (THREADS * vec);
  p.z_blocks = z != nullptr ? (z_cols + THREADS * vec - 1) / (THREADS * vec) : 0;
  const dim3 grid(p.u_blocks + p.z_blocks + (heads * (max_q_len < TOKENS ? max_q_len : TOKENS) + THREADS - 1) / THREADS, (max_q_len + TOKENS - 1) / TOKENS, entries);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == kF32 && wide) launch_prepare<float, 4>(p, grid, s);
  else if (dtype == kF32) launch_prepare<float, 1>(p, grid, s);
  else if (dtype == kBF16 && wide) launch_prepare<__nv_bfloat16, 4>(p, grid, s);
  else if (dtype == kBF16) launch_prepare<__nv_bfloat16, 1>(p, grid, s);
  else return fail(1, "ssm_prepare: unknown dtype %d", dtype);
  return check_launch("ssm_prepare");
}

// y float32 [tokens, groups * size] -> columns out_off .. of out [tokens, out_ld] in out_dtype.
PAE_EXPORT int pae_gated_group_norm(void* out, int out_ld, int out_off, const float* y, const float* gate, int gate_ld, int gate_off,
                                    const float* weight, int tokens, int groups, int size, int gate_first, float eps, float mult,
                                    int out_dtype, void* stream) {
  if (tokens == 0) return 0;
  if (groups < 1 || size < 1) return fail(2, "gated_group_norm: %d groups of %d channels", groups, size);
  if (out_off < 0 || out_off + groups * size > out_ld || gate_off < 0 || gate_off + groups * size > gate_ld)
    return fail(2, "gated_group_norm: %d channels from column %d of rows of %d, gates from %d of %d", groups * size, out_off, out_ld, gate_off, gate_ld);
  if (groups > 65535) return fail(3, "gated_group_norm: %d groups exceed one launch", groups);
  const GroupNorm p{y, gate, weight, out, groups, size, gate_ld, gate_off, out_ld, out_off, gate_first, eps, mult};
  const bool wide = ((size | gate_ld | gate_off | out_ld | out_off) & 3) == 0 && aligned16(y) && aligned16(gate) && aligned16(out);
  cudaStream_t s = (cudaStream_t)stream;
  if (out_dtype == kF32 && wide) launch_group_norm<float, 4>(p, tokens, s);
  else if (out_dtype == kF32) launch_group_norm<float, 1>(p, tokens, s);
  else if (out_dtype == kBF16 && wide) launch_group_norm<__nv_bfloat16, 4>(p, tokens, s);
  else if (out_dtype == kBF16) launch_group_norm<__nv_bfloat16, 1>(p, tokens, s);
  else return fail(1, "gated_group_norm: unknown dtype %d", out_dtype);
  return check_launch("gated_group_norm");
}

PAE_DEFINE_LAST_ERROR()

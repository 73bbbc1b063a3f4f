// What stands between a fused projection and attention, for mixers that norm and rotate their
// heads: per query and key head an optional RMS norm over the head's first channels with a
// weight shared by all heads (or one RMS norm over all query heads of the token at once, and one
// over all key heads, with a weight as long as the projection), a rotation of a span of the head
// by the step's table of cosines and sines, in either pairing, and the write of keys (and values)
// into their pages.
//
//   norm      y[i] = x[i] / sqrt(mean(x[0..span)^2) + eps) * w[i]      for i < span; the rest passes
//   or        y[h, i] = x[h, i] / sqrt(mean over all heads and channels of x^2 + eps) * w[h, i]   ("whole")
//   rotation  of channels [rot0, rot0 + dims): pair (i, i + dims/2) ("half") or (2i, 2i + 1)
//             ("interleaved"), i < dims/2:  (u, v) -> (u c_i - v s_i, v c_i + u s_i)
//   write     q -> q_out[token, head, :]; k -> keys[page, kv head, offset, :]; v likewise
//
// Query heads and key heads may differ in size, span and where their rotated channels start, so
// one launch serves grouped-query attention (all heads alike) and latent attention (query heads
// of unrotated + rotated channels; ONE key row per token that holds the normed latent and the
// shared rotated part; no values). The projection is float32 or the engine's element type; all
// arithmetic is float32 (the sum of squares double) and every result is rounded once.
//
// Also here: the table of cosines and sines with an amplitude, and the element-wise product of
// an attention's output with the sigmoid of a gate projection.
#include "common.cuh"

using namespace pae;

namespace {

struct HeadPrep {
  const void* proj;      // [tokens, ld]
  void* q_out;           // [tokens, heads, qd], a row every q_ld elements
  void* keys;            // [pages, kv_heads, page_size, kd]
  void* values;          // [pages, kv_heads, page_size, dv]
  const float* q_norm;   // [q_span] or null
  const float* k_norm;   // [k_span] or null
  const float* table;    // [tokens, dims]: cosines, then sines; null: no rotation
  const int* slots;      // [tokens]: page * page_size + offset, negative: nothing is written; null: no pages (or `direct`)
  int ld, q_ld, q_off, k_off, v_off;
  int heads, kv_heads, qd, kd, dv;
  int q_span, k_span, q_rot0, k_rot0, dims, interleaved, page_size;
  float eps;
  int whole;             // the norm's mean runs over all query (key) heads of the token; weights [heads, span]
  int direct;            // keys and values leave as plain rows [tokens, kv_heads, d], as the queries do
  int whole_kv_heads;    // the key heads that the mean runs over (kv_heads is 0 in a step that writes no page)
};

constexpr int WARPS = 4;

template <typename TI, typename TO>
__global__ void __launch_bounds__(WARPS * 32) head_prep_kernel(const HeadPrep p) {
  dependent_launch_prologue();
  extern __shared__ float rows[];              // [WARPS][widest head]
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int widest = max(max(p.qd, p.kd), p.dv);
  float* buf = rows + warp * widest;
  const TI* in = (const TI*)p.proj + (size_t)t * p.ld;
  const bool with_values = p.values != nullptr && p.dv > 0;
  const int units = p.heads + p.kv_heads * (with_values ? 2 : 1);
  int slot = -1;
  if (p.slots != nullptr) {
    slot = p.slots[t];
    if (slot >= 0 && !slot_in_pool(slot, p.page_size)) slot = -1;
  }
  if (p.direct) slot = t;                      // a page of one token each
  const int page = slot >= 0 ? slot / p.page_size : 0, offset = slot >= 0 ? slot - page * p.page_size : 0;
  const int half = p.dims >> 1;
  // "whole": the token's two sums of squares, by the whole block in an order that depends on
  // nothing but the sizes (so a token's result is the same in any batch)
  __shared__ double whole_sum[2][WARPS];
  float whole_inv[2] = {0.f, 0.f};
  if (p.whole) {
    for (int which = 0; which < 2; ++which) {
      const TI* src = in + (which == 0 ? p.q_off : p.k_off);
      // keys are normed whether or not the token has a page: the count is the model's, not the step's
      const int n = which == 0 ? (p.q_norm != nullptr ? p.heads * p.qd : 0) : (p.k_norm != nullptr ? p.whole_kv_heads * p.kd : 0);
      double squares = 0.0;
      for (int i = threadIdx.x; i < n; i += WARPS * 32) {
        const float v = to_float(src[i]);
        squares = fma((double)v, (double)v, squares);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) squares += __shfl_xor_sync(0xffffffffu, squares, o);
      if (lane == 0) whole_sum[which][warp] = squares;
    }
    __syncthreads();
    for (int which = 0; which < 2; ++which) {
      const int n = which == 0 ? p.heads * p.qd : p.whole_kv_heads * p.kd;
      double squares = 0.0;
      for (int w = 0; w < WARPS; ++w) squares += whole_sum[which][w];
      whole_inv[which] = n > 0 ? (float)(1.0 / sqrt(squares / (double)n + (double)p.eps)) : 0.f;
    }
  }
  for (int unit = blockIdx.y * WARPS + warp; unit < units; unit += WARPS * gridDim.y) {
    const bool is_q = unit < p.heads, is_k = !is_q && unit < p.heads + p.kv_heads;
    const int index = is_q ? unit : (is_k ? unit - p.heads : unit - p.heads - p.kv_heads);
    const int d = is_q ? p.qd : (is_k ? p.kd : p.dv);
    if (!is_q && slot < 0) continue;           // a key or value without a page is not wanted
    const TI* src = in + (is_q ? p.q_off : (is_k ? p.k_off : p.v_off)) + (size_t)index * d;
    const float* weight = is_q ? p.q_norm : (is_k ? p.k_norm : nullptr);
    const int span = is_q ? p.q_span : (is_k ? p.k_span : 0);
    if (p.whole && weight != nullptr) weight += (size_t)index * span;
    double squares = 0.0;
    for (int i = lane; i < d; i += 32) {
      const float v = to_float(src[i]);
      buf[i] = v;
      if (weight != nullptr && i < span) squares = fma((double)v, (double)v, squares);
    }
    if (p.whole && weight != nullptr) {
      const float inv = whole_inv[is_q ? 0 : 1];
      __syncwarp();
      for (int i = lane; i < span; i += 32) buf[i] = buf[i] * inv * weight[i];
    } else if (weight != nullptr && span > 0) {
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) squares += __shfl_xor_sync(0xffffffffu, squares, o);
      const float inv = (float)(1.0 / sqrt(squares / (double)span + (double)p.eps));
      __syncwarp();
      for (int i = lane; i < span; i += 32) buf[i] = buf[i] * inv * weight[i];
    }
    __syncwarp();
    if (p.table != nullptr && (is_q || is_k) && half > 0) {
      const int rot0 = is_q ? p.q_rot0 : p.k_rot0;
      const float* cs = p.table + (size_t)t * p.dims;
      for (int i = lane; i < half; i += 32) {
        const int a = rot0 + (p.interleaved ? 2 * i : i), b = rot0 + (p.interleaved ? 2 * i + 1 : i + half);
        float lo = buf[a], hi = buf[b];
        rotate_pair(lo, hi, cs[i], cs[half + i]);
        buf[a] = lo;
        buf[b] = hi;
      }
      __syncwarp();
    }
    TO* to;
    if (is_q)
      to = (TO*)p.q_out + (size_t)t * p.q_ld + (size_t)index * d;
    else
      to = (TO*)(is_k ? p.keys : p.values) + (((size_t)page * p.kv_heads + index) * p.page_size + offset) * d;
    for (int i = lane; i < d; i += 32) to[i] = from_float<TO>(buf[i]);
    __syncwarp();
  }
}

// The same without norms, for head sizes that split into pieces of 8 channels: a thread takes one piece
// of one head of one token, either 8 neighbouring channels or, of a span whose pairs are half a span
// apart, 4 channels and their 4 partners. No shared memory, 16-byte loads.
__device__ __forceinline__ void store4(float* to, const float* v) { *(float4*)to = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* to, const float* v) {
  uint2 packed;
  *(__nv_bfloat162*)&packed.x = __floats2bfloat162_rn(v[0], v[1]);
  *(__nv_bfloat162*)&packed.y = __floats2bfloat162_rn(v[2], v[3]);
  *(uint2*)to = packed;
}

template <typename TO>
__global__ void __launch_bounds__(256) head_rotate_kernel(const HeadPrep p, long long total) {
  dependent_launch_prologue();
  const long long at = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (at >= total) return;
  const int q_pieces = p.heads * (p.qd >> 3), k_pieces = p.kv_heads * (p.kd >> 3);
  const int v_pieces = p.values != nullptr ? p.kv_heads * (p.dv >> 3) : 0;
  const int per_token = q_pieces + k_pieces + v_pieces;
  const int t = (int)(at / per_token);
  int piece = (int)(at - (long long)t * per_token);
  const bool is_q = piece < q_pieces, is_k = !is_q && piece < q_pieces + k_pieces;
  piece -= is_q ? 0 : (is_k ? q_pieces : q_pieces + k_pieces);
  const int d = is_q ? p.qd : (is_k ? p.kd : p.dv);
  const int index = piece / (d >> 3), j = piece - index * (d >> 3);
  TO* to;
  if (is_q) {
    to = (TO*)p.q_out + (size_t)t * p.q_ld + (size_t)index * d;
  } else {
    int slot = p.direct ? t : p.slots[t];
    if (slot < 0 || (!p.direct && !slot_in_pool(slot, p.page_size))) return;
    const int page = slot / p.page_size, offset = slot - page * p.page_size;
    to = (TO*)(is_k ? p.keys : p.values) + (((size_t)page * p.kv_heads + index) * p.page_size + offset) * d;
  }
  const float* from = (const float*)p.proj + (size_t)t * p.ld + (is_q ? p.q_off : (is_k ? p.k_off : p.v_off)) + (size_t)index * d;
  const bool turns = p.table != nullptr && (is_q || is_k) && j < (p.dims >> 3);
  const int half = p.dims >> 1;
  const int a = turns && !p.interleaved ? 4 * j : 8 * j, b = turns && !p.interleaved ? half + 4 * j : 8 * j + 4;
  const float4 x4 = *(const float4*)(from + a), y4 = *(const float4*)(from + b);
  float x[4] = {x4.x, x4.y, x4.z, x4.w}, y[4] = {y4.x, y4.y, y4.z, y4.w};
  if (turns) {
    const float* cs = p.table + (size_t)t * p.dims + 4 * j;
    const float4 c4 = *(const float4*)cs, s4 = *(const float4*)(cs + half);
    const float c[4] = {c4.x, c4.y, c4.z, c4.w}, s[4] = {s4.x, s4.y, s4.z, s4.w};
    if (p.interleaved) {
      rotate_pair(x[0], x[1], c[0], s[0]);
      rotate_pair(x[2], x[3], c[1], s[1]);
      rotate_pair(y[0], y[1], c[2], s[2]);
      rotate_pair(y[2], y[3], c[3], s[3]);
    } else {
#pragma unroll
      for (int i = 0; i < 4; ++i) rotate_pair(x[i], y[i], c[i], s[i]);
    }
  }
  store4(to + a, x);
  store4(to + b, y);
}

bool aligned16(const void* ptr) { return (((uintptr_t)ptr) & 15) == 0; }

// table[t, i] = amplitude * cos(position[t] * inv_freq[i]), table[t, half + i] = amplitude * sin(same);
// the angle is one float32 product.
__global__ void rotary_table_amplitude_kernel(float* __restrict__ table, const int* __restrict__ positions,
                                              const float* __restrict__ inv_freq, int tokens, int half, float amplitude) {
  dependent_launch_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)tokens * half) return;
  const int t = (int)(i / half), f = (int)(i - (long long)t * half);
  const float angle = __fmul_rn((float)positions[t], inv_freq[f]);
  float s, c;
  sincosf(angle, &s, &c);
  table[(size_t)t * 2 * half + f] = c * amplitude;
  table[(size_t)t * 2 * half + half + f] = s * amplitude;
}

// out[t, out_off + c] = mult * x[t, c] * sigmoid(gate[t, gate_off + c / group]); the gate is a column
// range of a projection, one column for every `group` neighbouring channels (a head's size: a gate
// per head); the result is a column range of rows of out_ld elements.
struct GateOut {
  int width, out_ld, out_off, gate_ld, gate_off, group;
  float mult;
};

template <typename TX, typename TG>
__global__ void sigmoid_gate_kernel(TX* __restrict__ out, const TX* __restrict__ x, const TG* __restrict__ gate, long long total,
                                    const GateOut p) {
  dependent_launch_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const long long t = i / p.width;
  const int c = (int)(i - t * p.width);
  const float g = to_float(gate[t * p.gate_ld + p.gate_off + c / p.group]);
  out[t * p.out_ld + p.out_off + c] = from_float<TX>(p.mult * to_float(x[i]) / (1.f + expf(-g)));
}

// The same for bfloat16 x, a float32 gate per channel and everything aligned: four channels a thread.
__global__ void __launch_bounds__(256) sigmoid_gate4_kernel(__nv_bfloat16* __restrict__ out, const __nv_bfloat16* __restrict__ x,
                                                            const float* __restrict__ gate, long long quads, const GateOut p) {
  dependent_launch_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= quads) return;
  const int per_row = p.width >> 2;
  const long long t = i / per_row;
  const int c = (int)(i - t * per_row) * 4;
  const uint2 x4 = *(const uint2*)(x + t * p.width + c);
  const float4 g4 = *(const float4*)(gate + t * p.gate_ld + p.gate_off + c);
  const float2 lo = __bfloat1622float2(*(const __nv_bfloat162*)&x4.x), hi = __bfloat1622float2(*(const __nv_bfloat162*)&x4.y);
  uint2 packed;
  *(__nv_bfloat162*)&packed.x = __floats2bfloat162_rn(p.mult * lo.x / (1.f + expf(-g4.x)), p.mult * lo.y / (1.f + expf(-g4.y)));
  *(__nv_bfloat162*)&packed.y = __floats2bfloat162_rn(p.mult * hi.x / (1.f + expf(-g4.z)), p.mult * hi.y / (1.f + expf(-g4.w)));
  *(uint2*)(out + t * p.out_ld + p.out_off + c) = packed;
}

}  // namespace

// direct: keys and values go to plain rows [tokens, kv_heads, d] instead of pages.
// whole: the norms' means run over all heads at once (weights [heads * span]). in_dtype: the projection's element type; out_dtype: that of q_out and of the pages (0 float32, 1 bfloat16).
PAE_EXPORT int pae_head_prep(void* q_out, int q_ld, void* keys, void* values, const void* proj, int ld, int q_off, int k_off,
                             int v_off, int tokens, int heads, int kv_heads, int qd, int kd, int dv,
                             const float* q_norm, int q_span, const float* k_norm, int k_span, float eps,
                             const float* table, int dims, int interleaved, int q_rot0, int k_rot0, const int* slots,
                             int page_size, int whole, int direct, int in_dtype, int out_dtype, void* stream) {
  if (tokens == 0 || heads + kv_heads == 0) return 0;
  if (heads < 0 || kv_heads < 0 || qd < 0 || kd < 0 || dv < 0) return fail(2, "head_prep: a negative size");
  if (dims % 2) return fail(2, "head_prep: %d rotated channels are not pairs", dims);
  if (table != nullptr && ((heads > 0 && q_rot0 + dims > qd) || (kv_heads > 0 && k_rot0 + dims > kd)))
    return fail(2, "head_prep: %d rotated channels from %d and %d do not fit heads of %d and %d", dims, q_rot0, k_rot0, qd, kd);
  if (q_span > qd || k_span > kd) return fail(2, "head_prep: a norm over %d or %d channels of heads of %d and %d", q_span, k_span, qd, kd);
  if (kv_heads > 0 && (slots != nullptr || direct) && (keys == nullptr || (page_size < 1 && !direct))) return fail(2, "head_prep: slots without pages");
  if (heads > 0 && q_out == nullptr) return fail(2, "head_prep: query heads without an output");
  if (heads > 0 && q_ld < heads * qd) return fail(2, "head_prep: query rows of %d for %d heads of %d", q_ld, heads, qd);
  if (whole && ((q_norm != nullptr && q_span != qd) || (k_norm != nullptr && k_span != kd)))
    return fail(2, "head_prep: a norm over the whole projection covers every channel (%d of %d, %d of %d)", q_span, qd, k_span, kd);
  HeadPrep p{proj, q_out, keys, values, q_norm, k_norm, table, slots, ld, q_ld, q_off, k_off, v_off, heads,
             slots != nullptr || direct ? kv_heads : 0, qd, kd, dv, q_span, k_span, q_rot0, k_rot0, table != nullptr ? dims : 0,
             interleaved, direct || page_size < 1 ? 1 : page_size, eps, whole, direct, kv_heads};
  const int sizes = qd | (p.kv_heads > 0 ? kd | (values != nullptr ? dv : 0) : 0) | p.dims;
  if (in_dtype == kF32 && q_norm == nullptr && k_norm == nullptr && q_rot0 == 0 && k_rot0 == 0 && sizes % 8 == 0 &&
      ((ld | q_ld | q_off | k_off | v_off) & 3) == 0 && aligned16(proj) && aligned16(q_out) && aligned16(keys) && aligned16(values) &&
      aligned16(table)) {
    const long long total = (long long)tokens * (heads * (qd / 8) + p.kv_heads * (kd / 8 + (values != nullptr ? dv / 8 : 0)));
    const int threads = total < 64 * 1024 ? 64 : 256;
    const unsigned blocks = (unsigned)((total + threads - 1) / threads);
    if (out_dtype == kF32) launch_kernel(head_rotate_kernel<float>, blocks, threads, 0, (cudaStream_t)stream, p, total);
    else if (out_dtype == kBF16) launch_kernel(head_rotate_kernel<__nv_bfloat16>, blocks, threads, 0, (cudaStream_t)stream, p, total);
    else return fail(1, "head_prep: element type %d is not supported", out_dtype);
    return check_launch("head_prep");
  }
  const int widest = qd > kd ? (qd > dv ? qd : dv) : (kd > dv ? kd : dv);
  const size_t smem = sizeof(float) * WARPS * (size_t)widest;
  if (smem > 48 * 1024) return fail(2, "head_prep: heads of %d channels are too wide", widest);
  cudaStream_t s = (cudaStream_t)stream;
  using bf = __nv_bfloat16;
  const int key = in_dtype * 10 + out_dtype;
  // few tokens: a warp per head, so that a decode step's handful of tokens still fills some SMs
  const int units = heads + p.kv_heads * (values != nullptr && dv > 0 ? 2 : 1);
  const dim3 grid(tokens, tokens < 64 ? (units + WARPS - 1) / WARPS : 1);
  if (key == 0) launch_kernel(head_prep_kernel<float, float>, grid, WARPS * 32, smem, s, p);
  else if (key == 1) launch_kernel(head_prep_kernel<float, bf>, grid, WARPS * 32, smem, s, p);
  else if (key == 11) launch_kernel(head_prep_kernel<bf, bf>, grid, WARPS * 32, smem, s, p);
  else return fail(1, "head_prep: element types in=%d out=%d are not supported", in_dtype, out_dtype);
  return check_launch("head_prep");
}

PAE_EXPORT int pae_rotary_table_amplitude(float* table, const int* positions, const float* inv_freq, int tokens, int half,
                                          float amplitude, void* stream) {
  const long long n = (long long)tokens * half;
  if (n == 0) return 0;
  launch_kernel(rotary_table_amplitude_kernel, (unsigned)((n + 255) / 256), 256, 0, (cudaStream_t)stream, table, positions,
                inv_freq, tokens, half, amplitude);
  return check_launch("rotary_table_amplitude");
}

// x [tokens, width] and out [tokens, out_ld] (columns out_off .. out_off + width) in x_dtype; gate [tokens,
// gate_ld] in gate_dtype, columns gate_off .. gate_off + width / group.
PAE_EXPORT int pae_sigmoid_gate(void* out, int out_ld, int out_off, const void* x, const void* gate, int tokens, int width,
                                int gate_ld, int gate_off, int group, float mult, int x_dtype, int gate_dtype, void* stream) {
  const long long total = (long long)tokens * width;
  if (total == 0) return 0;
  if (group < 1 || width % group) return fail(2, "sigmoid_gate: rows of %d channels in groups of %d", width, group);
  if (gate_off < 0 || gate_off + width / group > gate_ld) return fail(2, "sigmoid_gate: columns %d..%d of rows of %d", gate_off, gate_off + width / group, gate_ld);
  if (out_off < 0 || out_off + width > out_ld) return fail(2, "sigmoid_gate: output columns %d..%d of rows of %d", out_off, out_off + width, out_ld);
  const GateOut p{width, out_ld, out_off, gate_ld, gate_off, group, mult};
  cudaStream_t s = (cudaStream_t)stream;
  using bf = __nv_bfloat16;
  const unsigned blocks = (unsigned)((total + 255) / 256);
  const int key = x_dtype * 10 + gate_dtype;
  if (key == 10 && group == 1 && ((width | out_ld | out_off | gate_ld | gate_off) & 3) == 0 && (((uintptr_t)x | (uintptr_t)out | (uintptr_t)gate) & 15) == 0) {
    launch_kernel(sigmoid_gate4_kernel, (unsigned)((total / 4 + 255) / 256), 256, 0, s, (bf*)out, (const bf*)x, (const float*)gate, total / 4, p);
    return check_launch("sigmoid_gate");
  }
  if (key == 0) launch_kernel(sigmoid_gate_kernel<float, float>, blocks, 256, 0, s, (float*)out, (const float*)x, (const float*)gate, total, p);
  else if (key == 10) launch_kernel(sigmoid_gate_kernel<bf, float>, blocks, 256, 0, s, (bf*)out, (const bf*)x, (const float*)gate, total, p);
  else if (key == 11) launch_kernel(sigmoid_gate_kernel<bf, bf>, blocks, 256, 0, s, (bf*)out, (const bf*)x, (const bf*)gate, total, p);
  else return fail(1, "sigmoid_gate: element types x=%d gate=%d are not supported", x_dtype, gate_dtype);
  return check_launch("sigmoid_gate");
}

PAE_DEFINE_LAST_ERROR()

// What stands between two sublayers of a decoder that norms what a sublayer leaves, not what it reads:
//
//   y      = sum_b scale_b * rms(y_b) * w_b        one output, or several branches side by side, each
//                                                  normed over the width with a weight of its own (or as it is)
//   x'     = x + mult * rms(y) * post_w            the norm after the sublayer and the residual sum
//   read   = x' in the engine's element type       what the next sublayer reads,
//            or rms(x') * read_w in it             or the model's last norm
//
// with rms(v) = v / sqrt(mean(v^2) + eps). A branch may be the planes of a split product, which are added
// in their order first. Every piece is optional, and a launch with the pieces that a caller has is what
// runs: the sum of branches alone, the residual alone, the rounding alone. A block owns a row. Rows of up
// to 8,192 columns that split into aligned 16-byte pieces, with one or two branches, stay in registers,
// all of their loads asked for before the first sum; any other row stays in shared memory between the
// passes, where a thread only ever touches its own columns. The stream and all arithmetic are float32 (sums
// of squares double), every read is rounded once.
#include "common.cuh"

using namespace pae;

namespace {

constexpr int MAX_BRANCHES = 4;

struct PostNorm {
  const float* x;                       // [rows, width] or null: x' = y
  float* x_new;                         // [rows, width] or null
  void* read;                           // [rows, width] or null
  const float* y[MAX_BRANCHES];         // [planes, rows, width]
  const float* w[MAX_BRANCHES];         // [width] or null: the branch is added as it is
  float scale[MAX_BRANCHES];
  int planes[MAX_BRANCHES];
  int branches;                         // 0: nothing is added
  const float* post_w;                  // [width] or null: y is added as it is
  const float* read_w;                  // [width] or null: x' as it is
  float branch_eps, post_eps, read_eps, mult;
  int width;
  long long total;
};

// The sum of a double per thread over the block; `scratch` holds one per warp.
__device__ __forceinline__ double row_sum(double v, double* scratch) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int warps = blockDim.x >> 5;
  __syncthreads();                       // scratch may still be read from the call before
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = v;
  __syncthreads();
  double total = 0.0;
  for (int i = 0; i < warps; ++i) total += scratch[i];     // every thread adds in the same order
  return total;
}

// Rounded step by step, so that every form of the kernel gives the same bits.
__device__ __forceinline__ float normed(float v, float inv, float w) { return __fmul_rn(__fmul_rn(v, inv), w); }

template <int VEC>
struct Piece {
  float v[VEC];
};
template <int VEC>
__device__ __forceinline__ Piece<VEC> get(const float* from) {
  Piece<VEC> p;
  if (VEC == 4) {
    const float4 f = *(const float4*)from;
    p.v[0] = f.x, p.v[1 % VEC] = f.y, p.v[2 % VEC] = f.z, p.v[3 % VEC] = f.w;
  } else {
    p.v[0] = *from;
  }
  return p;
}
template <int VEC>
__device__ __forceinline__ void put(float* to, const Piece<VEC>& p) {
  if (VEC == 4)
    *(float4*)to = make_float4(p.v[0], p.v[1 % VEC], p.v[2 % VEC], p.v[3 % VEC]);
  else
    *to = p.v[0];
}
template <int VEC>
__device__ __forceinline__ void put(__nv_bfloat16* to, const Piece<VEC>& p) {
  if (VEC == 4) {
    uint2 packed;
    *(__nv_bfloat162*)&packed.x = __floats2bfloat162_rn(p.v[0], p.v[1 % VEC]);
    *(__nv_bfloat162*)&packed.y = __floats2bfloat162_rn(p.v[2 % VEC], p.v[3 % VEC]);
    *(uint2*)to = packed;
  } else {
    *to = __float2bfloat16_rn(p.v[0]);
  }
}

// A piece of a branch: its planes added in their order, eight of them asked for at a time.
template <int VEC>
__device__ __forceinline__ Piece<VEC> branch_piece(const float* y, int planes, long long total) {
  Piece<VEC> s = get<VEC>(y);
  for (int k = 1; k < planes; k += 8) {
    Piece<VEC> more[8];
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (k + j < planes) more[j] = get<VEC>(y + (size_t)(k + j) * total);
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (k + j < planes)
#pragma unroll
        for (int e = 0; e < VEC; ++e) s.v[e] += more[j].v[e];
  }
  return s;
}

template <typename TO, int VEC>
__global__ void __launch_bounds__(1024) post_norm_kernel(const PostNorm p) {
  dependent_launch_prologue();
  extern __shared__ __align__(16) float row[];      // [max(branches, 1)][width]
  __shared__ double scratch[32];
  const int width = p.width, step = blockDim.x * VEC, c0 = threadIdx.x * VEC;
  const size_t at = (size_t)blockIdx.x * width;
  const double part = 1.0 / (double)width;
  auto inverse = [&](double squares, float eps) { return 1.f / sqrtf((float)fma(row_sum(squares, scratch), part, (double)eps)); };
  float inv[MAX_BRANCHES];
  for (int b = 0; b < p.branches; ++b) {
    double squares = 0.0;
    for (int c = c0; c < width; c += step) {
      const Piece<VEC> s = branch_piece<VEC>(p.y[b] + at + c, p.planes[b], p.total);
#pragma unroll
      for (int e = 0; e < VEC; ++e) squares = fma((double)s.v[e], (double)s.v[e], squares);
      put<VEC>(row + (size_t)b * width + c, s);
    }
    inv[b] = p.w[b] != nullptr || (p.branches == 1 && p.post_w != nullptr) ? inverse(squares, p.w[b] != nullptr ? p.branch_eps : p.post_eps) : 0.f;
  }
  // a single output that is not normed as a branch has its sum of squares already
  const bool single = p.branches == 1 && p.w[0] == nullptr && p.scale[0] == 1.f;
  float post = single ? inv[0] : 0.f;
  if (p.branches > 0 && !single) {
    double squares = 0.0;
    for (int c = c0; c < width; c += step) {
      Piece<VEC> v;
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] = 0.f;
      for (int b = 0; b < p.branches; ++b) {
        const Piece<VEC> s = get<VEC>(row + (size_t)b * width + c);
        if (p.w[b] != nullptr) {
          const Piece<VEC> w = get<VEC>(p.w[b] + c);
#pragma unroll
          for (int e = 0; e < VEC; ++e) v.v[e] = fmaf(p.scale[b], normed(s.v[e], inv[b], w.v[e]), v.v[e]);
        } else {
#pragma unroll
          for (int e = 0; e < VEC; ++e) v.v[e] = fmaf(p.scale[b], s.v[e], v.v[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) squares = fma((double)v.v[e], (double)v.v[e], squares);
      put<VEC>(row + c, v);
    }
    if (p.post_w != nullptr) post = inverse(squares, p.post_eps);
  }
  double squares = 0.0;
  TO* read = (TO*)p.read + at;
  for (int c = c0; c < width; c += step) {
    Piece<VEC> x;
    if (p.x != nullptr) {
      x = get<VEC>(p.x + at + c);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) x.v[e] = 0.f;
    }
    if (p.branches > 0) {
      const Piece<VEC> v = get<VEC>(row + c);
      if (p.post_w != nullptr) {
        const Piece<VEC> w = get<VEC>(p.post_w + c);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x.v[e] = fmaf(p.mult, normed(v.v[e], post, w.v[e]), x.v[e]);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x.v[e] = fmaf(p.mult, v.v[e], x.v[e]);
      }
    }
    if (p.x_new != nullptr) put<VEC>(p.x_new + at + c, x);
    if (p.read == nullptr) continue;
    if (p.read_w == nullptr) {
      put<VEC>(read + c, x);
    } else {
#pragma unroll
      for (int e = 0; e < VEC; ++e) squares = fma((double)x.v[e], (double)x.v[e], squares);
      put<VEC>(row + c, x);
    }
  }
  if (p.read == nullptr || p.read_w == nullptr) return;
  const float last = inverse(squares, p.read_eps);
  for (int c = c0; c < width; c += step) {
    Piece<VEC> x = get<VEC>(row + c);
    const Piece<VEC> w = get<VEC>(p.read_w + c);
#pragma unroll
    for (int e = 0; e < VEC; ++e) x.v[e] = normed(x.v[e], last, w.v[e]);
    put<VEC>(read + c, x);
  }
}

// The row in registers: PER pieces of four columns a thread, BRANCHES outputs.
template <typename TO, int PER, int BRANCHES>
__global__ void __launch_bounds__(PER <= 4 ? 512 : 256) post_norm_row_kernel(const PostNorm p) {
  dependent_launch_prologue();
  constexpr int AHEAD = PER == 1 ? 8 : (PER == 2 ? 4 : 1);      // planes asked for at a time (few rows have planes, and few pieces a thread)
  __shared__ double scratch[3][BRANCHES][16];      // a set per sum: one barrier each
  const int width = p.width, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const size_t at = (size_t)blockIdx.x * width;
  const int c0 = threadIdx.x * 4, step = blockDim.x * 4;
  const double part = 1.0 / (double)width;
  auto inverse = [&](double total, float eps) { return 1.f / sqrtf((float)fma(total, part, (double)eps)); };
  Piece<4> y[BRANCHES][PER], x[PER];
#pragma unroll
  for (int b = 0; b < BRANCHES; ++b)
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (c0 + i * step < width) y[b][i] = get<4>(p.y[b] + at + c0 + i * step);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    x[i].v[0] = x[i].v[1] = x[i].v[2] = x[i].v[3] = 0.f;
    if (p.x != nullptr && c0 + i * step < width) x[i] = get<4>(p.x + at + c0 + i * step);
  }
  double squares[BRANCHES];
#pragma unroll
  for (int b = 0; b < BRANCHES; ++b) {
    const float* from = p.y[b] + at + c0;
    for (int k = 1; k < p.planes[b]; k += AHEAD) {      // the planes in their order
      Piece<4> more[AHEAD][PER];
#pragma unroll
      for (int j = 0; j < AHEAD; ++j)
#pragma unroll
        for (int i = 0; i < PER; ++i)
          if (k + j < p.planes[b] && c0 + i * step < width) more[j][i] = get<4>(from + (size_t)(k + j) * p.total + i * step);
#pragma unroll
      for (int j = 0; j < AHEAD; ++j)
#pragma unroll
        for (int i = 0; i < PER; ++i)
          if (k + j < p.planes[b] && c0 + i * step < width)
#pragma unroll
            for (int e = 0; e < 4; ++e) y[b][i].v[e] += more[j][i].v[e];
    }
    squares[b] = 0.0;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (c0 + i * step < width)
#pragma unroll
        for (int e = 0; e < 4; ++e) squares[b] = fma((double)y[b][i].v[e], (double)y[b][i].v[e], squares[b]);
  }
  auto share = [&](double v, int set, int b) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    if (lane == 0) scratch[set][b][warp] = v;
  };
  auto total = [&](int set, int b) {
    double sum = 0.0;
    for (int w = 0; w < warps; ++w) sum += scratch[set][b][w];      // every thread adds in the same order
    return sum;
  };
  const bool own_norms = p.w[0] != nullptr || (BRANCHES > 1 && p.w[BRANCHES - 1] != nullptr);      // some branch has a norm of its own
  const bool plain = BRANCHES == 1 && !own_norms && p.scale[0] == 1.f;
  if (own_norms || (plain && p.post_w != nullptr)) {
#pragma unroll
    for (int b = 0; b < BRANCHES; ++b) share(squares[b], 0, b);
    __syncthreads();
  }
  float post = 0.f;
  if (plain) {
    if (p.post_w != nullptr) post = inverse(total(0, 0), p.post_eps);
  } else {
    double sum = 0.0;
    float inv[BRANCHES];
#pragma unroll
    for (int b = 0; b < BRANCHES; ++b) inv[b] = p.w[b] != nullptr ? inverse(total(0, b), p.branch_eps) : 1.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      if (c0 + i * step >= width) break;
      Piece<4> v;
#pragma unroll
      for (int e = 0; e < 4; ++e) v.v[e] = 0.f;
#pragma unroll
      for (int b = 0; b < BRANCHES; ++b) {
        if (p.w[b] != nullptr) {
          const Piece<4> w = get<4>(p.w[b] + c0 + i * step);
#pragma unroll
          for (int e = 0; e < 4; ++e) v.v[e] = fmaf(p.scale[b], normed(y[b][i].v[e], inv[b], w.v[e]), v.v[e]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) v.v[e] = fmaf(p.scale[b], y[b][i].v[e], v.v[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) sum = fma((double)v.v[e], (double)v.v[e], sum);
      y[0][i] = v;
    }
    if (p.post_w != nullptr) {
      share(sum, 1, 0);
      __syncthreads();
      post = inverse(total(1, 0), p.post_eps);
    }
  }
  double sum = 0.0;
  TO* read = (TO*)p.read + at;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int c = c0 + i * step;
    if (c >= width) break;
    if (p.post_w != nullptr) {
      const Piece<4> w = get<4>(p.post_w + c);
#pragma unroll
      for (int e = 0; e < 4; ++e) x[i].v[e] = fmaf(p.mult, normed(y[0][i].v[e], post, w.v[e]), x[i].v[e]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) x[i].v[e] = fmaf(p.mult, y[0][i].v[e], x[i].v[e]);
    }
    if (p.x_new != nullptr) put<4>(p.x_new + at + c, x[i]);
    if (p.read == nullptr) continue;
    if (p.read_w == nullptr) {
      put<4>(read + c, x[i]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) sum = fma((double)x[i].v[e], (double)x[i].v[e], sum);
    }
  }
  if (p.read == nullptr || p.read_w == nullptr) return;
  share(sum, 2, 0);
  __syncthreads();
  const float last = inverse(total(2, 0), p.read_eps);
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int c = c0 + i * step;
    if (c >= width) break;
    const Piece<4> w = get<4>(p.read_w + c);
#pragma unroll
    for (int e = 0; e < 4; ++e) x[i].v[e] = normed(x[i].v[e], last, w.v[e]);
    put<4>(read + c, x[i]);
  }
}

// The stream rounded, nothing else: the first sublayer's read.
__global__ void __launch_bounds__(256) round_kernel(__nv_bfloat16* __restrict__ out, const float* __restrict__ x, long long total) {
  dependent_launch_prologue();
  const long long at = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (at >= total) return;
  put<4>(out + at, get<4>(x + at));
  if (at + 4 < total) put<4>(out + at + 4, get<4>(x + at + 4));
}

template <typename TO, int BRANCHES>
int launch_row(const PostNorm& p, int rows, cudaStream_t s) {
  const int pieces = p.width / 4;
  // many rows: a few warps a row, so that an SM holds many; few rows: as many threads as there are pieces
  const int threads = rows > 64 ? (pieces <= 1024 ? 128 : 256) : (pieces <= 128 ? 128 : pieces <= 256 ? 256 : 512);
  switch ((pieces + threads - 1) / threads) {
    case 1: launch_kernel(post_norm_row_kernel<TO, 1, BRANCHES>, rows, threads, 0, s, p); break;
    case 2: launch_kernel(post_norm_row_kernel<TO, 2, BRANCHES>, rows, threads, 0, s, p); break;
    case 3: launch_kernel(post_norm_row_kernel<TO, 3, BRANCHES>, rows, threads, 0, s, p); break;
    case 4: launch_kernel(post_norm_row_kernel<TO, 4, BRANCHES>, rows, threads, 0, s, p); break;
    case 5:
    case 6: launch_kernel(post_norm_row_kernel<TO, 6, BRANCHES>, rows, threads, 0, s, p); break;
    default: launch_kernel(post_norm_row_kernel<TO, 8, BRANCHES>, rows, threads, 0, s, p); break;
  }
  return check_launch("post_norm");
}

constexpr size_t SMEM_MOST = 200 * 1024;

bool aligned16(const void* ptr) { return (((uintptr_t)ptr) & 15) == 0; }

template <typename TO, int VEC>
int launch(const PostNorm& p, int rows, int threads, size_t bytes, cudaStream_t s) {
  static bool raised = false;
  if (bytes > 48 * 1024 && !raised) {
    cudaError_t err = cudaFuncSetAttribute(post_norm_kernel<TO, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM_MOST);
    if (err != cudaSuccess) return fail(100, "post_norm: %s", cudaGetErrorString(err));
    raised = true;
  }
  launch_kernel(post_norm_kernel<TO, VEC>, rows, threads, bytes, s, p);
  return check_launch("post_norm");
}

}  // namespace

// Up to four branches (y0 first; planes, weight or null, and scale of each). x, x_new, read, post_w and read_w
// may be null. read_dtype: the element type of `read` (0 float32, 1 bfloat16).
PAE_EXPORT int pae_post_norm(float* x_new, void* read, const float* x, int branches, const float* y0, const float* y1, const float* y2,
                             const float* y3, int planes0, int planes1, int planes2, int planes3, const float* w0, const float* w1,
                             const float* w2, const float* w3, float scale0, float scale1, float scale2, float scale3, float branch_eps,
                             const float* post_w, float post_eps, float mult, const float* read_w, float read_eps, int rows, int width,
                             int read_dtype, void* stream) {
  if (rows == 0 || width == 0) return 0;
  if (branches < 0 || branches > MAX_BRANCHES) return fail(2, "post_norm: %d branches (0 to %d)", branches, MAX_BRANCHES);
  if (x == nullptr && branches == 0) return fail(2, "post_norm: neither a stream nor a branch");
  if (read_dtype != kF32 && read_dtype != kBF16) return fail(1, "post_norm: unknown dtype %d", read_dtype);
  PostNorm p{x, x_new, read, {y0, y1, y2, y3}, {w0, w1, w2, w3}, {scale0, scale1, scale2, scale3}, {planes0, planes1, planes2, planes3},
             branches, post_w, read_w, branch_eps, post_eps, read_eps, mult, width, (long long)rows * width};
  bool wide = width % 4 == 0 && aligned16(x_new) && aligned16(read) && aligned16(x) && aligned16(post_w) && aligned16(read_w);
  for (int b = 0; b < MAX_BRANCHES; ++b) {
    if (b < branches && (p.y[b] == nullptr || p.planes[b] < 1)) return fail(2, "post_norm: branch %d has %d planes", b, p.planes[b]);
    wide = wide && aligned16(p.y[b]) && aligned16(p.w[b]);
  }
  if (wide && branches == 0 && read_w == nullptr && x_new == nullptr && read_dtype == kBF16) {
    launch_kernel(round_kernel, (unsigned)((p.total / 4 + 511) / 512), 256, 0, (cudaStream_t)stream, (__nv_bfloat16*)read, x, p.total);
    return check_launch("post_norm_round");
  }
  if (wide && width <= 8192 && (branches == 1 || branches == 2)) {
    cudaStream_t s = (cudaStream_t)stream;
    if (read_dtype == kF32) return branches == 1 ? launch_row<float, 1>(p, rows, s) : launch_row<float, 2>(p, rows, s);
    return branches == 1 ? launch_row<__nv_bfloat16, 1>(p, rows, s) : launch_row<__nv_bfloat16, 2>(p, rows, s);
  }
  const size_t bytes = sizeof(float) * (size_t)(branches > 1 ? branches : 1) * width;
  if (bytes > SMEM_MOST) return fail(2, "post_norm: %d rows of %d do not fit shared memory", branches, width);
  const int pieces = wide ? width / 4 : width;
  int threads = 64;
  while (threads < pieces && threads < (rows < 64 ? 1024 : 512)) threads *= 2;
  cudaStream_t s = (cudaStream_t)stream;
  if (read_dtype == kF32) return wide ? launch<float, 4>(p, rows, threads, bytes, s) : launch<float, 1>(p, rows, threads, bytes, s);
  return wide ? launch<__nv_bfloat16, 4>(p, rows, threads, bytes, s) : launch<__nv_bfloat16, 1>(p, rows, threads, bytes, s);
}

PAE_DEFINE_LAST_ERROR()

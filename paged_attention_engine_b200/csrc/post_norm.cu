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
// runs: the sum of branches alone, the residual alone, the rounding alone. A block owns a row and keeps it
// in shared memory between the passes; a thread only ever touches its own columns there, so the barriers
// are the ones inside the sums. The stream and all arithmetic are float32 (sums of squares double),
// every read is rounded once.
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
  auto inverse = [&](double squares, float eps) { return (float)(1.0 / sqrt(row_sum(squares, scratch) / (double)width + (double)eps)); };
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
          for (int e = 0; e < VEC; ++e) v.v[e] += p.scale[b] * (s.v[e] * inv[b] * w.v[e]);
        } else {
#pragma unroll
          for (int e = 0; e < VEC; ++e) v.v[e] += p.scale[b] * s.v[e];
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
        for (int e = 0; e < VEC; ++e) x.v[e] += p.mult * (v.v[e] * post * w.v[e]);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) x.v[e] += p.mult * v.v[e];
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
    for (int e = 0; e < VEC; ++e) x.v[e] = x.v[e] * last * w.v[e];
    put<VEC>(read + c, x);
  }
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

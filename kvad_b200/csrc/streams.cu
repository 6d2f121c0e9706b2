// A residual stream held as several copies side by side (hyper-connections): what a sublayer reads, what it leaves, and
// the norm in between, in one pass over the rows.
//
//   with an owed result y:   x'_t = sum_s mix[s, t] x_s + share[t] y          (all copies at once from the old ones)
//   without:                 x'_t = x_t
//   u = sum_t read[t] x'_t                                                     (`read` absent: the plain sum)
//   out = norm(u):  centred: (u - mean) / sqrt(mean((u - mean)^2) + eps) * gain + bias;  else u / sqrt(mean(u^2) + eps) * gain + bias
//
// The copies are [copies][rows, width], 32-bit; a stride of 0 between copies means that all of them are still the one
// tensor they start from.  With all rows walked the new copies are written and y is cleared for the next sublayer to add
// into; with a row list only `out` is written (the head, which is the last to read).  Everything is 32-bit; the order of a
// row's sums depends on the width alone.
#include "common.cuh"

using namespace kvad;

namespace {

constexpr int MAX_COPIES = 16;

struct StreamArgs {
  const float* x; int64_t x_stride;        // the copies as they are (stride between copies, 0: one tensor)
  float* x_out; int64_t out_stride;        // where the new copies go (may be x)
  float* y;                                // the owed result, or null
  const float* mix; const float* share;    // [copies, copies] from | to, [copies]
  const float* read;                       // [copies] or null
  const int* rows;                         // or null: all rows, and the copies are written
  const void* gain; const void* bias; int params_f32;
  void* out;
  int n_rows, width, copies, centred;
  float eps;
};

__device__ __forceinline__ void store4(float* o, float4 v) { *reinterpret_cast<float4*>(o) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* o, float4 v) {
  __nv_bfloat162 p[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
  *reinterpret_cast<uint2*>(o) = *reinterpret_cast<const uint2*>(p);
}

__device__ __forceinline__ float4 load_params4(const void* p, int c, int is_f32) {
  if (is_f32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + c);
  const uint2 q = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p) + c);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&q);
  const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
  return make_float4(a.x, a.y, b.x, b.y);
}

__device__ __forceinline__ float4 fma4(float w, float4 a, float4 c) {
  return make_float4(fmaf(w, a.x, c.x), fmaf(w, a.y, c.y), fmaf(w, a.z, c.z), fmaf(w, a.w, c.w));
}

// Sum over the block's warps, in warp order; `met` holds a float per warp and is used once per launch.
__device__ __forceinline__ float meet(float v, float* met) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) met[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = met[0];
  for (int w = 1; w < (int)(blockDim.x >> 5); ++w) t += met[w];
  return t;
}

// A block per row, the row's weighted sum in registers: NI pieces of four columns a thread.
template <typename T, int S, int NI>
__global__ void __launch_bounds__(256) streams_norm_kernel(const StreamArgs a) {
  __shared__ float met[2][8];
  pdl_launch_dependents();
  float mix[S][S], share[S], read[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    read[s] = a.read ? a.read[s] : 1.f;
    share[s] = a.y ? a.share[s] : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = a.y ? a.mix[s * S + t] : (s == t ? 1.f : 0.f);
  }
  float4 g[NI], b[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    g[i] = c < a.width ? load_params4(a.gain, c, a.params_f32) : make_float4(0.f, 0.f, 0.f, 0.f);
    b[i] = c < a.width && a.bias ? load_params4(a.bias, c, a.params_f32) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  const int64_t row = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  const float* xr = a.x + row * a.width;
  float* yr = a.y ? a.y + row * a.width : nullptr;
  const bool one = a.x_stride == 0;
  float4 u[NI];
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < a.width) {
      float4 x[S];
      x[0] = *reinterpret_cast<const float4*>(xr + c);
#pragma unroll
      for (int s = 1; s < S; ++s) x[s] = one ? x[0] : *reinterpret_cast<const float4*>(xr + s * a.x_stride + c);
      if (yr != nullptr) {
        const float4 y = *reinterpret_cast<const float4*>(yr + c);
#pragma unroll
        for (int t = 0; t < S; ++t) {
          float4 n = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int s = 0; s < S; ++s) n = fma4(mix[s][t], x[s], n);
          n = fma4(share[t], y, n);
          u[i] = fma4(read[t], n, u[i]);
          if (a.rows == nullptr) *reinterpret_cast<float4*>(a.x_out + t * a.out_stride + row * a.width + c) = n;
        }
        if (a.rows == nullptr) *reinterpret_cast<float4*>(yr + c) = make_float4(0.f, 0.f, 0.f, 0.f);
      } else {
#pragma unroll
        for (int t = 0; t < S; ++t) u[i] = fma4(read[t], x[t], u[i]);
      }
      sum += a.centred ? (u[i].x + u[i].y) + (u[i].z + u[i].w) : 0.f;
    }
  }
  const float mean = a.centred ? meet(sum, met[0]) / (float)a.width : 0.f;
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    if ((int)(threadIdx.x + i * blockDim.x) * 4 < a.width) {
      u[i] = make_float4(u[i].x - mean, u[i].y - mean, u[i].z - mean, u[i].w - mean);
      sq = fmaf(u[i].x, u[i].x, fmaf(u[i].y, u[i].y, fmaf(u[i].z, u[i].z, fmaf(u[i].w, u[i].w, sq))));
    }
  }
  const float inv = 1.0f / sqrtf(meet(sq, met[1]) / (float)a.width + a.eps);
  T* o = reinterpret_cast<T*>(a.out) + (int64_t)blockIdx.x * a.width;
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c < a.width)
      store4(o + c, make_float4(fmaf(u[i].x * inv, g[i].x, b[i].x), fmaf(u[i].y * inv, g[i].y, b[i].y),
                                fmaf(u[i].z * inv, g[i].z, b[i].z), fmaf(u[i].w * inv, g[i].w, b[i].w)));
  }
}

// Any width, any number of copies up to MAX_COPIES: the row's weighted sum in shared memory, an entry at a time.
template <typename T>
__global__ void __launch_bounds__(256) streams_norm_any_kernel(const StreamArgs a) {
  extern __shared__ float u[];
  __shared__ float met[2][8];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  const int S = a.copies;
  float sum = 0.f;
  for (int c = threadIdx.x; c < a.width; c += blockDim.x) {
    float x[MAX_COPIES];
    for (int s = 0; s < S; ++s) x[s] = a.x[s * a.x_stride + row * a.width + c];
    const float y = a.y ? a.y[row * a.width + c] : 0.f;
    float v = 0.f;
    for (int t = 0; t < S; ++t) {
      float n = x[t];
      if (a.y != nullptr) {
        n = 0.f;
        for (int s = 0; s < S; ++s) n = fmaf(a.mix[s * S + t], x[s], n);
        n = fmaf(a.share[t], y, n);
        if (a.rows == nullptr) a.x_out[t * a.out_stride + row * a.width + c] = n;
      }
      v = fmaf(a.read ? a.read[t] : 1.f, n, v);
    }
    if (a.y != nullptr && a.rows == nullptr) a.y[row * a.width + c] = 0.f;
    u[c] = v;
    sum += v;
  }
  const float mean = a.centred ? meet(sum, met[0]) / (float)a.width : 0.f;
  float sq = 0.f;
  for (int c = threadIdx.x; c < a.width; c += blockDim.x) {
    const float d = u[c] - mean;
    sq = fmaf(d, d, sq);
  }
  const float inv = 1.0f / sqrtf(meet(sq, met[1]) / (float)a.width + a.eps);
  T* o = reinterpret_cast<T*>(a.out) + (int64_t)blockIdx.x * a.width;
  for (int c = threadIdx.x; c < a.width; c += blockDim.x)
    o[c] = from_f32<T>(fmaf((u[c] - mean) * inv, load_param(a.gain, c, a.params_f32), a.bias ? load_param(a.bias, c, a.params_f32) : 0.f));
}

template <typename T, int S>
int launch_copies(const StreamArgs& a, cudaStream_t stream) {
  int threads = (a.width / 4 + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  const int pieces = (a.width / 4 + threads - 1) / threads;
  const dim3 grid(a.n_rows), block(threads);
  if (pieces <= 1) kvad_launch(streams_norm_kernel<T, S, 1>, grid, block, 0, stream, a);
  else if (pieces <= 2) kvad_launch(streams_norm_kernel<T, S, 2>, grid, block, 0, stream, a);
  else if (pieces <= 4) kvad_launch(streams_norm_kernel<T, S, 4>, grid, block, 0, stream, a);
  else kvad_launch(streams_norm_kernel<T, S, 8>, grid, block, 0, stream, a);
  return 0;
}

template <typename T>
int launch_streams(const StreamArgs& a, cudaStream_t stream) {
  const uintptr_t at = reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.x_out) | reinterpret_cast<uintptr_t>(a.y) |
                       reinterpret_cast<uintptr_t>(a.gain) | reinterpret_cast<uintptr_t>(a.bias) | reinterpret_cast<uintptr_t>(a.out);
  const bool pieces = a.width % 4 == 0 && a.width <= 8192 && a.x_stride % 4 == 0 && a.out_stride % 4 == 0 && (at & 15) == 0;
  if (pieces && a.copies == 1) return launch_copies<T, 1>(a, stream);
  if (pieces && a.copies == 2) return launch_copies<T, 2>(a, stream);
  if (pieces && a.copies == 3) return launch_copies<T, 3>(a, stream);
  if (pieces && a.copies == 4) return launch_copies<T, 4>(a, stream);
  const size_t smem = (size_t)a.width * sizeof(float);
  if (smem > 48 * 1024) KVAD_FAIL(KVAD_ERR_UNSUPPORTED, "streams_norm: %d copies of rows of %d entries are above this kernel's limits", a.copies, a.width);
  kvad_launch(streams_norm_any_kernel<T>, dim3(a.n_rows), dim3(256), smem, stream, a);
  return 0;
}

}  // namespace

// x: the copies [copies][rows, width] `x_stride` floats apart (0: all of them are one tensor).  y (may be null: nothing is owed)
// with mix [copies, copies] (from, to) and share [copies]; the new copies go to x_out (`out_stride` apart), y is cleared -
// both only without a row list.  read [copies] or null (ones).  out [n_rows, width] = norm of the weighted sum.
KVAD_EXPORT int kvad_streams_norm(int out_dtype, const float* x, int64_t x_stride, float* x_out, int64_t out_stride, float* y,
                                  const float* mix, const float* share, const float* read, const int* rows, const void* gain,
                                  const void* bias, int params_f32, int centred, void* out, int n_rows, int width, int copies,
                                  float eps, cudaStream_t stream) {
  KVAD_REQUIRE(n_rows >= 0 && width > 0 && copies >= 1 && copies <= MAX_COPIES, "streams_norm: bad sizes rows=%d width=%d copies=%d (1..%d)", n_rows,
               width, copies, MAX_COPIES);
  KVAD_REQUIRE(x && gain && out, "streams_norm: a pointer is missing");
  KVAD_REQUIRE(y == nullptr || (mix && share && (rows != nullptr || x_out)), "streams_norm: an owed result needs its mix, its shares and a place for the new copies");
  KVAD_REQUIRE(x_stride != 0 || x_out != x || y == nullptr || copies == 1, "streams_norm: copies that are still one tensor cannot be written in place");
  if (n_rows == 0) return KVAD_OK;
  StreamArgs a;
  a.x = x; a.x_stride = x_stride; a.x_out = x_out; a.out_stride = out_stride; a.y = y; a.mix = mix; a.share = share; a.read = read; a.rows = rows;
  a.gain = gain; a.bias = bias; a.params_f32 = params_f32; a.out = out; a.n_rows = n_rows; a.width = width; a.copies = copies; a.centred = centred;
  a.eps = eps;
  int status;
  if (out_dtype == KVAD_DTYPE_F32) status = launch_streams<float>(a, stream);
  else if (out_dtype == KVAD_DTYPE_BF16) status = launch_streams<__nv_bfloat16>(a, stream);
  else KVAD_FAIL(KVAD_ERR_UNSUPPORTED, "streams_norm: unknown dtype %d", out_dtype);
  if (status != 0) return status;
  KVAD_CHECK_LAUNCH("streams_norm");
  return KVAD_OK;
}

KVAD_DEFINE_LAST_ERROR()

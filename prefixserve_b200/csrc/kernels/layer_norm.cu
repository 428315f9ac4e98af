// The residual sum and one or two layer norms of its result, a block per row:
//
//   v = h + pending                                     (pending optional; the stream h becomes v with ``update``)
//   y = (v - mean(v)) / sqrt(mean((v - mean(v))^2) + eps)
//   x1 = y * gain1 + shift1,  x2 = y * gain2 + shift2   (the second optional: two sublayers that read one stream through
//                                                        norms of their own share the sum, the mean and the variance)
//
// With ``rows`` only the named rows are computed (the last use of the stream).  All arithmetic is float32; the variance is the
// mean of the squared deviations, taken in a second pass over the row.  layer_norm_vec_kernel holds the row in registers, eight
// channels a thread and run.
#include "common.cuh"

namespace {

constexpr int LN_THREADS = 256;

template <typename T, int N>
struct alignas(sizeof(T) * N) Run {
  T v[N];
};

// The sum over the block of one number a thread, in the same order for every thread and batch.
__device__ __forceinline__ float block_sum(float a, float* scratch) {
  a = warp_sum(a);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  if (lane == 0) scratch[warp] = a;
  __syncthreads();
  float total = 0.f;
  for (int w = 0; w < warps; ++w) total += scratch[w];
  __syncthreads();
  return total;
}

template <typename T>
struct NormArgs {
  float* h;
  const T* pending;
  const float *gain1, *shift1, *gain2, *shift2;
  const int32_t* rows;
  T *x1, *x2;
  int W, update;
  float eps;
};

template <typename T, int VPT>
__global__ void __launch_bounds__(LN_THREADS) layer_norm_vec_kernel(const NormArgs<T> p) {
  __shared__ float scratch[LN_THREADS / 32];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  const size_t r = (size_t)(p.rows ? p.rows[i] : i) * p.W;
  float v[VPT][8];
  float sum = 0.f;
#pragma unroll
  for (int c = 0; c < VPT; ++c) {
    const int j = (c * blockDim.x + threadIdx.x) * 8;
    if (j >= p.W) continue;
    const Run<float, 8> h = *reinterpret_cast<const Run<float, 8>*>(p.h + r + j);
#pragma unroll
    for (int k = 0; k < 8; ++k) v[c][k] = h.v[k];
    if (p.pending) {
      const Run<T, 8> d = *reinterpret_cast<const Run<T, 8>*>(p.pending + r + j);
#pragma unroll
      for (int k = 0; k < 8; ++k) v[c][k] += to_float<T>(d.v[k]);
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) sum += v[c][k];
    if (p.update) {
      Run<float, 8> o;
#pragma unroll
      for (int k = 0; k < 8; ++k) o.v[k] = v[c][k];
      *reinterpret_cast<Run<float, 8>*>(p.h + r + j) = o;
    }
  }
  const float mean = block_sum(sum, scratch) / (float)p.W;
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < VPT; ++c) {
    if ((c * blockDim.x + threadIdx.x) * 8 >= p.W) continue;
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      v[c][k] -= mean;
      ss = fmaf(v[c][k], v[c][k], ss);
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)p.W + p.eps);
  auto put = [&](int c, int j, const float* gain, const float* shift, T* x) {
    const Run<float, 8> g = *reinterpret_cast<const Run<float, 8>*>(gain + j), b = *reinterpret_cast<const Run<float, 8>*>(shift + j);
    Run<T, 8> o;
#pragma unroll
    for (int k = 0; k < 8; ++k) o.v[k] = from_float<T>(fmaf(v[c][k] * inv, g.v[k], b.v[k]));
    *reinterpret_cast<Run<T, 8>*>(x + (size_t)i * p.W + j) = o;
  };
#pragma unroll
  for (int c = 0; c < VPT; ++c) {
    const int j = (c * blockDim.x + threadIdx.x) * 8;
    if (j >= p.W) continue;
    put(c, j, p.gain1, p.shift1, p.x1);
    if (p.x2) put(c, j, p.gain2, p.shift2, p.x2);
  }
}

template <typename T>
__global__ void __launch_bounds__(LN_THREADS) layer_norm_kernel(const NormArgs<T> p) {
  __shared__ float scratch[LN_THREADS / 32];
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x;
  const size_t r = (size_t)(p.rows ? p.rows[i] : i) * p.W;
  auto value = [&](int j) { return p.h[r + j] + (p.pending ? to_float<T>(p.pending[r + j]) : 0.f); };
  float sum = 0.f;
  for (int j = threadIdx.x; j < p.W; j += blockDim.x) sum += value(j);
  const float mean = block_sum(sum, scratch) / (float)p.W;
  float ss = 0.f;
  for (int j = threadIdx.x; j < p.W; j += blockDim.x) {
    const float d = value(j) - mean;
    ss = fmaf(d, d, ss);
  }
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)p.W + p.eps);
  for (int j = threadIdx.x; j < p.W; j += blockDim.x) {  // a thread reads and writes its own channels only
    const float v = value(j);
    if (p.update) p.h[r + j] = v;
    const float y = (v - mean) * inv;
    p.x1[(size_t)i * p.W + j] = from_float<T>(fmaf(y, p.gain1[j], p.shift1[j]));
    if (p.x2) p.x2[(size_t)i * p.W + j] = from_float<T>(fmaf(y, p.gain2[j], p.shift2[j]));
  }
}

}  // namespace

// (h, pending, dtype, gain1, shift1, gain2, shift2, rows, x1, x2, n_rows, W, eps, update, stream); pending, rows and the second
// norm (gain2, shift2, x2 together) may be null
PSB_API int psb_add_layer_norm(void* h, const void* pending, int dtype, const void* gain1, const void* shift1, const void* gain2,
                               const void* shift2, const void* rows, void* x1, void* x2, int n_rows, int W, float eps, int update,
                               cudaStream_t stream) {
  if (n_rows < 0 || W < 1 || !(eps > 0.f)) PSB_REFUSE("add_layer_norm: bad sizes rows=%d W=%d eps=%g", n_rows, W, eps);
  if (!gain1 || !shift1 || !x1 || ((x2 == nullptr) != (gain2 == nullptr)) || ((x2 == nullptr) != (shift2 == nullptr)))
    PSB_REFUSE("add_layer_norm: every norm needs its gain, its shift and its rows");
  if (rows && update) PSB_REFUSE("add_layer_norm: chosen rows leave the stream as it is");
  if (n_rows == 0) return 0;
  const uintptr_t every = (uintptr_t)h | (uintptr_t)pending | (uintptr_t)gain1 | (uintptr_t)shift1 | (uintptr_t)gain2 | (uintptr_t)shift2 |
                          (uintptr_t)x1 | (uintptr_t)x2;
  const bool vec = W % 8 == 0 && (every & 31) == 0 && W <= 8 * 4 * LN_THREADS;
  PSB_DISPATCH_DTYPE(dtype, T, {
    const NormArgs<T> p{(float*)h, (const T*)pending, (const float*)gain1, (const float*)shift1, (const float*)gain2, (const float*)shift2,
                        (const int32_t*)rows, (T*)x1, (T*)x2, W, update, eps};
    const int threads = W <= 8 * 128 ? 128 : LN_THREADS;
    const int vpt = (W / 8 + threads - 1) / threads;
    if (!vec) psb_launch(layer_norm_kernel<T>, dim3(n_rows), dim3(threads), 0, stream, p);
    else if (vpt <= 1) psb_launch(layer_norm_vec_kernel<T, 1>, dim3(n_rows), dim3(threads), 0, stream, p);
    else if (vpt == 2) psb_launch(layer_norm_vec_kernel<T, 2>, dim3(n_rows), dim3(threads), 0, stream, p);
    else psb_launch(layer_norm_vec_kernel<T, 4>, dim3(n_rows), dim3(threads), 0, stream, p);
  });
  PSB_LAUNCH_CHECK("add_layer_norm");
  return 0;
}

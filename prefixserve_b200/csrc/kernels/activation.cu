// Activations of a feed-forward without a gate branch, out = act(x) element by element, float32 arithmetic (rows of the result
// may be runs of columns of wider ones):
//   silu, gelu_tanh (as in the gated kernels), and xielu with two learned numbers (p, q):
//     z > 0:  softplus(p) z^2 + z/2
//     z <= 0: (1/2 + softplus(q)) (exp(z) - 1 - z) + z/2
//   and relu2: max(z, 0)^2.
// poly_norm looks at a whole row: with N dividing a row by its root mean square, a N(z) + b N(z^2) + c N(z^3) + e with four
// learned numbers (a block per row; the three sums in one pass, the row kept in registers where it fits).
// soft_cap: logits <- cap * tanh(logits / cap), in place.
#include "common.cuh"

namespace {

enum : int { UNARY_SILU = 0, UNARY_GELU_TANH = 1, UNARY_XIELU = 2, UNARY_RELU2 = 3 };

__device__ __forceinline__ float relu2f_(float z) { z = fmaxf(z, 0.f); return z * z; }

__device__ __forceinline__ float softplusf_(float x) { return log1pf(expf(-fabsf(x))) + fmaxf(x, 0.f); }

template <typename T>
__global__ void unary_act_kernel(const T* __restrict__ x, T* __restrict__ out, size_t total, int code,
                                 const float* __restrict__ params, size_t cols, size_t ldo) {
  pdl_trigger();
  pdl_wait();
  float ap = 0.f, aq = 0.f;
  if (code == UNARY_XIELU) {
    ap = softplusf_(params[0]);
    aq = 0.5f + softplusf_(params[1]);
  }
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const float z = to_float<T>(x[i]);
    float v;
    if (code == UNARY_XIELU) v = z > 0.f ? ap * z * z + 0.5f * z : aq * (expm1f(z) - z) + 0.5f * z;
    else if (code == UNARY_RELU2) v = relu2f_(z);
    else v = gate_act(z, code);
    out[cols == ldo ? i : i / cols * ldo + i % cols] = from_float<T>(v);
  }
}

// Eight bfloat16 elements a thread (16-byte loads and stores).
__global__ void unary_act_vec_kernel(const __nv_bfloat16* __restrict__ x, __nv_bfloat16* __restrict__ out, size_t vecs, int code,
                                     const float* __restrict__ params, size_t cols8, size_t ldo8) {
  pdl_trigger();
  pdl_wait();
  float ap = 0.f, aq = 0.f;
  if (code == UNARY_XIELU) {
    ap = softplusf_(params[0]);
    aq = 0.5f + softplusf_(params[1]);
  }
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < vecs; i += (size_t)gridDim.x * blockDim.x) {
    const uint4 raw = reinterpret_cast<const uint4*>(x)[i];
    const __nv_bfloat162* in2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
    uint4 o4;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o4);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 z = __bfloat1622float2(in2[k]);
      float a, b;
      if (code == UNARY_XIELU) {
        a = z.x > 0.f ? ap * z.x * z.x + 0.5f * z.x : aq * (expm1f(z.x) - z.x) + 0.5f * z.x;
        b = z.y > 0.f ? ap * z.y * z.y + 0.5f * z.y : aq * (expm1f(z.y) - z.y) + 0.5f * z.y;
      } else if (code == UNARY_RELU2) {
        a = relu2f_(z.x);
        b = relu2f_(z.y);
      } else {
        a = gate_act(z.x, code);
        b = gate_act(z.y, code);
      }
      o2[k] = __floats2bfloat162_rn(a, b);
    }
    reinterpret_cast<uint4*>(out)[cols8 == ldo8 ? i : i / cols8 * ldo8 + i % cols8] = o4;
  }
}

// out = x * gate, element by element: gate float32 (a sigmoid that somebody has already taken), the product in float32
template <typename TX, typename TO>
__global__ void gate_mul_kernel(const TX* __restrict__ x, const float* __restrict__ gate, TO* __restrict__ out, size_t total) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x)
    out[i] = from_float<TO>(to_float<TX>(x[i]) * gate[i]);
}

template <typename T, int N>
struct alignas(sizeof(T) * N) ActRun {
  T v[N];
};

constexpr int POLY_THREADS = 256;

// N elements a thread and run; KEEP runs a thread stay in registers between the two passes, later ones are read again.
template <typename T, int N, int KEEP>
__global__ void __launch_bounds__(POLY_THREADS)
poly_norm_kernel(const T* __restrict__ z, T* __restrict__ out, const float* __restrict__ act, int W, float eps) {
  __shared__ float sums[3][POLY_THREADS / 32];
  pdl_trigger();
  pdl_wait();
  const T* row = z + (size_t)blockIdx.x * W;
  T* dst = out + (size_t)blockIdx.x * W;
  ActRun<T, N> held[KEEP];
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  auto add = [&](const ActRun<T, N>& x) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const float v = to_float<T>(x.v[i]), v2 = v * v, v3 = v2 * v;
      s1 += v2;
      s2 = fmaf(v2, v2, s2);
      s3 = fmaf(v3, v3, s3);
    }
  };
#pragma unroll
  for (int c = 0; c < KEEP; ++c) {
    const int j = (c * POLY_THREADS + threadIdx.x) * N;
    if (j < W) {
      held[c] = *reinterpret_cast<const ActRun<T, N>*>(row + j);
      add(held[c]);
    }
  }
  for (int j = (KEEP * POLY_THREADS + threadIdx.x) * N; j < W; j += POLY_THREADS * N) add(*reinterpret_cast<const ActRun<T, N>*>(row + j));
  s1 = warp_sum(s1);
  s2 = warp_sum(s2);
  s3 = warp_sum(s3);
  if ((threadIdx.x & 31) == 0) {
    sums[0][threadIdx.x >> 5] = s1;
    sums[1][threadIdx.x >> 5] = s2;
    sums[2][threadIdx.x >> 5] = s3;
  }
  __syncthreads();
  s1 = s2 = s3 = 0.f;
  for (int w = 0; w < POLY_THREADS / 32; ++w) {
    s1 += sums[0][w];
    s2 += sums[1][w];
    s3 += sums[2][w];
  }
  const float a = act[0] / sqrtf(s1 / (float)W + eps), b = act[1] / sqrtf(s2 / (float)W + eps), c3 = act[2] / sqrtf(s3 / (float)W + eps);
  const float e = act[3];
  auto value = [&](const ActRun<T, N>& x) {
    ActRun<T, N> o;
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const float v = to_float<T>(x.v[i]);
      o.v[i] = from_float<T>(fmaf(v, fmaf(v, fmaf(v, c3, b), a), e));
    }
    return o;
  };
#pragma unroll
  for (int c = 0; c < KEEP; ++c) {
    const int j = (c * POLY_THREADS + threadIdx.x) * N;
    if (j < W) *reinterpret_cast<ActRun<T, N>*>(dst + j) = value(held[c]);
  }
  for (int j = (KEEP * POLY_THREADS + threadIdx.x) * N; j < W; j += POLY_THREADS * N)
    *reinterpret_cast<ActRun<T, N>*>(dst + j) = value(*reinterpret_cast<const ActRun<T, N>*>(row + j));
}

template <int N>
__global__ void soft_cap_kernel(float* __restrict__ x, size_t runs, float cap) {
  pdl_trigger();
  pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < runs; i += (size_t)gridDim.x * blockDim.x) {
    ActRun<float, N> v = reinterpret_cast<const ActRun<float, N>*>(x)[i];
#pragma unroll
    for (int k = 0; k < N; ++k) v.v[k] = cap * tanhf(v.v[k] / cap);
    reinterpret_cast<ActRun<float, N>*>(x)[i] = v;
  }
}

}  // namespace

// (z [rows, W], dtype, out, act float32 [4], rows, W, eps, stream)
PSB_API int psb_poly_norm(const void* z, int dtype, void* out, const void* act, int rows, int W, float eps, cudaStream_t stream) {
  if (rows < 0 || W < 1 || !act || !(eps > 0.f)) PSB_REFUSE("poly_norm: bad arguments rows=%d W=%d", rows, W);
  if (rows == 0) return 0;
  PSB_DISPATCH_DTYPE(dtype, T, {
    const bool runs = W % 8 == 0 && (((uintptr_t)z | (uintptr_t)out) % (8 * sizeof(T))) == 0;
    if (runs && W <= 2 * POLY_THREADS * 8)
      psb_launch(poly_norm_kernel<T, 8, 2>, dim3(rows), dim3(POLY_THREADS), 0, stream, (const T*)z, (T*)out, (const float*)act, W, eps);
    else if (runs)
      psb_launch(poly_norm_kernel<T, 8, 4>, dim3(rows), dim3(POLY_THREADS), 0, stream, (const T*)z, (T*)out, (const float*)act, W, eps);
    else
      psb_launch(poly_norm_kernel<T, 1, 4>, dim3(rows), dim3(POLY_THREADS), 0, stream, (const T*)z, (T*)out, (const float*)act, W, eps);
  });
  PSB_LAUNCH_CHECK("poly_norm");
  return 0;
}

// (logits float32, total, cap, stream): in place
PSB_API int psb_soft_cap(void* x, long long total, float cap, cudaStream_t stream) {
  if (total < 0 || !(cap > 0.f)) PSB_REFUSE("soft_cap: bad arguments total=%lld cap=%f", total, (double)cap);
  if (total == 0) return 0;
  const bool wide = total % 4 == 0 && ((uintptr_t)x & 15) == 0;
  const long long runs = wide ? total / 4 : total, blocks = (runs + 255) / 256;
  const dim3 grid((unsigned)(blocks > 148 * 16 ? 148 * 16 : blocks));
  if (wide) psb_launch(soft_cap_kernel<4>, grid, dim3(256), 0, stream, (float*)x, (size_t)runs, cap);
  else psb_launch(soft_cap_kernel<1>, grid, dim3(256), 0, stream, (float*)x, (size_t)runs, cap);
  PSB_LAUNCH_CHECK("soft_cap");
  return 0;
}

// (x, x_dtype, gate float32, out, out_dtype, total, stream)
PSB_API int psb_gate_mul(const void* x, int x_dtype, const void* gate, void* out, int out_dtype, long long total, cudaStream_t stream) {
  if (total < 0) PSB_REFUSE("gate_mul: negative size");
  if (total == 0) return 0;
  const long long blocks = (total + 255) / 256;
  PSB_DISPATCH_DTYPE(x_dtype, TX, {
    PSB_DISPATCH_DTYPE(out_dtype, TO, {
      psb_launch(gate_mul_kernel<TX, TO>, dim3((unsigned)(blocks > 148 * 16 ? 148 * 16 : blocks)), dim3(256), 0, stream,
                 (const TX*)x, (const float*)gate, (TO*)out, (size_t)total);
    });
  });
  PSB_LAUNCH_CHECK("gate_mul");
  return 0;
}

// (x [total / cols, cols], dtype, out in rows ldo numbers apart, total, cols, ldo, code, params or null, stream)
PSB_API int psb_unary_act(const void* x, int dtype, void* out, long long total, long long cols, long long ldo, int code,
                          const void* params, cudaStream_t stream) {
  if (cols < 1 || ldo < cols || total % cols) PSB_REFUSE("unary_act: %lld numbers in rows of %lld, %lld apart", total, cols, ldo);
  if (total < 0) PSB_REFUSE("unary_act: negative size");
  if (code < 0 || code > UNARY_RELU2) PSB_REFUSE("unary_act: activation code %d is not built", code);
  if (code == UNARY_XIELU && !params) PSB_REFUSE("unary_act: xielu needs its two numbers");
  if (total == 0) return 0;
  if (dtype == PSB_BF16 && cols % 8 == 0 && ldo % 8 == 0 && (((uintptr_t)x | (uintptr_t)out) & 15) == 0) {
    const long long vecs = total / 8, vblocks = (vecs + 255) / 256;
    psb_launch(unary_act_vec_kernel, dim3((unsigned)(vblocks > 148 * 16 ? 148 * 16 : vblocks)), dim3(256), 0, stream,
               (const __nv_bfloat16*)x, (__nv_bfloat16*)out, (size_t)vecs, code, (const float*)params, (size_t)(cols / 8), (size_t)(ldo / 8));
    PSB_LAUNCH_CHECK("unary_act");
    return 0;
  }
  const long long blocks = (total + 255) / 256;
  PSB_DISPATCH_DTYPE(dtype, T, {
    psb_launch(unary_act_kernel<T>, dim3((unsigned)(blocks > 65535 * 16 ? 65535 * 16 : blocks)), dim3(256), 0, stream,
               (const T*)x, (T*)out, (size_t)total, code, (const float*)params, (size_t)cols, (size_t)ldo);
  });
  PSB_LAUNCH_CHECK("unary_act");
  return 0;
}

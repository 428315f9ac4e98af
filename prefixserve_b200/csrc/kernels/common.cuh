// Shared helpers for the sm_100a kernels: element types, error reporting, and
// the C ABI conventions.  Every entry point returns 0 on success; otherwise it
// has left a message for psb_last_error() and launched nothing (or the launch
// itself failed).
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>

#include <cstdint>
#include <cstdio>

#define PSB_API extern "C" __attribute__((visibility("default")))

enum PsbDtype : int { PSB_F32 = 0, PSB_BF16 = 1 };

void psb_set_error(const char* fmt, ...);

#define PSB_REFUSE(...)          \
  do {                           \
    psb_set_error(__VA_ARGS__);  \
    return 1;                    \
  } while (0)

#define PSB_LAUNCH_CHECK(name)                                                   \
  do {                                                                           \
    cudaError_t e_ = cudaGetLastError();                                         \
    if (e_ != cudaSuccess) {                                                     \
      psb_set_error("%s: launch failed: %s", name, cudaGetErrorString(e_));      \
      return 2;                                                                  \
    }                                                                            \
  } while (0)

// ---- programmatic dependent launch ---------------------------------------------------------------------------
// A decode step is a chain of some hundred short kernels, each waiting for the one before.  Launched with the
// programmatic-serialization attribute, a kernel may start while its predecessor is still draining: everything
// before pdl_wait() (index arithmetic, loads of weights and of the step's read-only inputs) overlaps with the
// predecessor; nothing the predecessor writes is read, and nothing is written, before pdl_wait() returns (it
// returns once the whole predecessor grid has finished and its writes are visible).  Every thread executes
// pdl_wait() before it exits, so that "this grid finished" always implies "its predecessor finished".  Without the
// launch attribute both instructions do nothing.
__device__ __forceinline__ void pdl_trigger() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

extern int psb_pdl_enabled;  // set through psb_set_pdl()

template <typename Kernel, typename... Args>
inline cudaError_t psb_launch(Kernel kernel, dim3 grid, dim3 block, size_t smem, cudaStream_t stream, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  if (psb_pdl_enabled) {
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
  }
  return cudaLaunchKernelEx(&cfg, kernel, args...);
}

// A function attribute (more than 48 KB of dynamic shared memory) has to be set once on every device that runs the
// kernel.  One of these per call site: get() is false until set() has been called with the same device current.
struct PsbPerDevice {
  static constexpr int kMaxDevices = 64;
  bool done[kMaxDevices] = {};
  static int current() {
    int d = 0;
    if (cudaGetDevice(&d) != cudaSuccess || d < 0 || d >= kMaxDevices) return -1;
    return d;
  }
  bool get() const {
    const int d = current();
    return d >= 0 && done[d];
  }
  void set() {
    const int d = current();
    if (d >= 0) done[d] = true;
  }
};

// (x1, x2) turned by the angle whose cosine and sine are given.  Written with explicit roundings, so that every
// kernel that rotates (the rotary kernels, the projection that rotates in its epilogue) rounds alike whatever the
// compiler would make of the plain expression around it.
__device__ __forceinline__ void rotate_pair(float x1, float x2, float cs, float sn, float& o1, float& o2) {
  o1 = __fmaf_rn(x1, cs, -__fmul_rn(x2, sn));
  o2 = __fmaf_rn(x2, cs, __fmul_rn(x1, sn));
}

// What a fused projection needs to finish the job of the rotary kernel (rope.cu) in its own epilogue: W is the
// [queries; keys; values] matrix with the rows of every query and key head reordered so that a 16-row tile holds
// 8 elements of the head's first half and the 8 elements they are rotated with (stored index 16b+j <-> natural
// index 8b+j, stored 16b+8+j <-> natural D/2+8b+j).  Queries go to q_out [M, hq, D] and keys to the cache in that
// stored order (a dot product does not care, as long as both sides agree); values in natural order.
struct RopeArgs {
  const int32_t* positions;   // [M] absolute position of each token
  const int32_t* token_item;  // [M] row of the page table
  const int32_t* table;       // [items, table_width] page ids
  const float* cos_t;         // [max_positions, D/2], null: no rotation
  const float* sin_t;
  __nv_bfloat16* kv;          // [num_pages, 2, hkv, page_size, D]
  __nv_bfloat16* q_out;       // [M, hq, D]
  int table_width, hq, hkv, D, page_shift, num_pages, max_positions;
};

// The activation of a gated feed-forward, act(gate) * up, by code: SiLU (prefixserve/model/llama.py:121 of
// PrefixServe, the only one that architecture uses) and the tanh form of GELU.  Every kernel that applies the
// activation takes the code; entry points refuse codes that are not listed here.
enum PsbAct : int { PSB_ACT_SILU = 0, PSB_ACT_GELU_TANH = 1 };
inline bool psb_activation_known(int code) { return code == PSB_ACT_SILU || code == PSB_ACT_GELU_TANH; }
__device__ __forceinline__ float gate_act(float g, int act) {
  if (act == PSB_ACT_GELU_TANH) return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g)));
  return g / (1.f + expf(-g));
}

// The same functions where the result is rounded to bfloat16 anyway (epilogues of the tensor-core products): the tanh form of
// GELU as z * sigmoid(2u), u = sqrt(2/pi) (z + 0.044715 z^3), since (1 + tanh u) / 2 = sigmoid(2u).
__device__ __forceinline__ float quick_act(float z, int act) {
  const float e = act == PSB_ACT_GELU_TANH ? 1.5957691216057308f * z * fmaf(0.044715f * z, z, 1.f) : z;
  return __fdividef(z, 1.f + __expf(-e));
}

// A gated feed-forward whose two branches are clipped before they meet: g = min(gate, limit), u = clamp(up, -limit, limit),
// value = g * sigmoid(alpha * g) * (u + offset).  It has numbers of its own, so it is no PsbAct code that every entry
// point takes: kernels that know it receive PSB_ACT_CLIPPED together with a GluClip.
constexpr int PSB_ACT_CLIPPED = 2;
struct GluClip {
  float limit, alpha, offset;
};
__device__ __forceinline__ float clipped_gate_value(float g, float u, const GluClip& c) {
  g = fminf(g, c.limit);
  u = fminf(fmaxf(u, -c.limit), c.limit);
  return g / (1.f + expf(-c.alpha * g)) * (u + c.offset);
}
// act(gate) * up for a PsbAct code, or the clipped form
__device__ __forceinline__ float gated_value(float g, float u, int act, const GluClip& c) {
  return act == PSB_ACT_CLIPPED ? clipped_gate_value(g, u, c) : gate_act(g, act) * u;
}

template <typename T>
__device__ __forceinline__ float to_float(T v);
template <>
__device__ __forceinline__ float to_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_float<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_float(float v);
template <>
__device__ __forceinline__ float from_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// A sink joins a finished softmax: one more term in the denominator, with a score of its own and no value.  ``e`` is
// the exponent the row's sum ``l`` and its accumulated values refer to (l = sum of 2^(x - e)) and ``s`` the sink's score,
// both in powers of two (natural scores times log2 e); -inf for a row that saw no key.  Returns what the accumulated
// values are multiplied by in place of 1 / l.  The larger of e and s is taken out first, so neither term overflows.
__device__ __forceinline__ float sink_quotient2(float e, float l, float s) {
  const float top = fmaxf(e, s);
  const float a = exp2f(e - top);  // 0 from -inf
  return a / fmaf(l, a, exp2f(s - top));
}
constexpr float PSB_LOG2E = 1.4426950408889634f;

// Calls f.template operator()<T>() with T chosen by a PsbDtype code.
#define PSB_DISPATCH_DTYPE(code, T, ...)                       \
  if ((code) == PSB_F32) { using T = float; __VA_ARGS__ }      \
  else if ((code) == PSB_BF16) { using T = __nv_bfloat16; __VA_ARGS__ } \
  else PSB_REFUSE("unknown dtype code %d", (int)(code))

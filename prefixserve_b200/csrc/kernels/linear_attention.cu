// Gated linear attention: a matrix state S [dim, vdim] per request and head that forgets key channel by key channel,
//
//     S <- diag(alpha_t) S + k_t v_t^T,    o_t = S^T q_t * scale,
//
// all of it float32.  Queries, keys and values are read where the layer's input product left them (rows ``ld`` numbers
// apart: [q: H dim | k: H dim | v: H vdim | ...]), alpha is float32 [T, H, dim], S lies in the request's slot [H, dim, vdim].
//
// The columns of S never meet.  R lanes of a warp hold NC columns between them (PER rows of each a lane, in registers; lane r
// holds rows in runs of four, 4 R apart, so that the lanes' reads of a token's vectors lie side by side, and what a lane
// reads of a token serves NC columns), a warp carries 32 / R * NC columns, and the NC read-outs of a token are finished by a
// butterfly among the R lanes in which each round halves the columns a lane still sums.  The order of every sum depends on
// the sizes only, never on the batch.  What a run of tokens brings is copied to shared memory (cp.async, in the types it
// has) one run ahead of the arithmetic.
//
// A step S -> diag(alpha) S + k v^T is a map S -> diag(A) S + B, and such maps compose.  Long portions are therefore cut
// into chunks of ``chunk`` tokens that run side by side:
//   linear_attention_kernel<.., true>   every chunk but a portion's last: A [dim] and B [dim, vdim] from a zero state;
//   linear_attention_starts_kernel      per portion, chunk by chunk: the state every chunk starts from (over B);
//   linear_attention_kernel<.., false>  every chunk from its start, with read-outs; the last one leaves the slot's state.
// A portion of one chunk takes the last kernel alone, from and to the slot.
//
// normed_readout_kernel (a warp per token and head): o / sqrt(mean(o^2) + eps) * gain[vdim] * gate, rounded to the compute
// type; the gate is read as it is, through silu or through a sigmoid; the gain is shared by the heads or each head has its own.
#include "common.cuh"

namespace {

constexpr int LA_WARPS = 4;
constexpr int LA_STAGE = 8;  // tokens a stage

__device__ __forceinline__ void la_copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void la_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void la_wait() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// The chunk a block works on: chunks are numbered through the step's items in order.  False beyond the last.
__device__ __forceinline__ bool find_chunk(const int32_t* __restrict__ item_start, int items, int chunk, int at, int& item, int& t0,
                                           int& t1, bool& only, bool& last) {
  for (int i = 0; i < items; ++i) {
    const int a = item_start[i], b = item_start[i + 1];
    const int n = (b - a + chunk - 1) / chunk;
    if (at < n) {
      item = i;
      t0 = a + at * chunk;
      t1 = min(b, t0 + chunk);
      only = n == 1;
      last = at == n - 1;
      return true;
    }
    at -= n;
  }
  return false;
}

template <int PER, int R>
__device__ __forceinline__ int row_of(int r, int e) {  // the row of S that is lane r's e-th
  return (e >> 2) * (4 * R) + r * 4 + (e & 3);
}

template <int PER, int R>
__device__ __forceinline__ void lane_vector(const float* v, int r, float (&o)[PER]) {
#pragma unroll
  for (int e = 0; e < PER; e += 4) {
    const float4 a = *reinterpret_cast<const float4*>(v + row_of<PER, R>(r, e));
    o[e] = a.x; o[e + 1] = a.y; o[e + 2] = a.z; o[e + 3] = a.w;
  }
}
template <int PER, int R>
__device__ __forceinline__ void lane_vector(const __nv_bfloat16* v, int r, float (&o)[PER]) {
#pragma unroll
  for (int e = 0; e < PER; e += 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(v + row_of<PER, R>(r, e));
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    o[e] = a.x; o[e + 1] = a.y; o[e + 2] = b.x; o[e + 3] = b.y;
  }
}

template <typename T, int PER, int R, int NC>
struct LaSizes {
  static constexpr int RP = PER * R, COLS = 32 / R * NC, BC = LA_WARPS * COLS;
  // bytes of a token in a stage: q and k (RP of type T each), alpha (RP floats), values (BC of type T)
  static constexpr int K_AT = RP * (int)sizeof(T), A_AT = 2 * K_AT, V_AT = A_AT + RP * 4, BYTES = V_AT + BC * (int)sizeof(T);
  static constexpr int SMEM = 2 * LA_STAGE * BYTES;
  static_assert(PER % 4 == 0 && (NC == 4 || NC == 2) && BC * sizeof(T) % 16 == 0 && K_AT % 16 == 0, "runs start on 16 bytes");
};

template <typename T, int PER, int R, int NC, bool LOCAL>
__global__ void __launch_bounds__(LA_WARPS * 32)
linear_attention_kernel(const T* __restrict__ proj, long long ld, const float* __restrict__ alpha, float* __restrict__ state,
                        long long slot_floats, const int32_t* __restrict__ item_start, const int32_t* __restrict__ slots,
                        float* __restrict__ local_b, float* __restrict__ local_a, float* __restrict__ o, int items, int H, int dim,
                        int vdim, int num_slots, int chunk, float scale) {
  using Z = LaSizes<T, PER, R, NC>;
  constexpr int RP = Z::RP, BC = Z::BC, EPP = 16 / (int)sizeof(T);  // EPP: elements of a 16-byte piece
  extern __shared__ __align__(16) unsigned char staged[];  // [2][LA_STAGE] tokens; zeros beyond dim and vdim
  pdl_trigger();
  pdl_wait();
  int item, t0, t1;
  bool only, last;
  if (!find_chunk(item_start, items, chunk, blockIdx.z, item, t0, t1, only, last)) return;
  if (LOCAL && last) return;
  const int h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane % R;
  const int col0 = blockIdx.x * BC, in_block = warp * Z::COLS + lane / R * NC, col = col0 + in_block;
  int slot = slots[item];
  slot = slot < 0 ? 0 : (slot >= num_slots ? num_slots - 1 : slot);
  float* S = state + (size_t)slot * slot_floats + (size_t)h * dim * vdim;
  float* B = local_b ? local_b + ((size_t)blockIdx.z * H + h) * dim * vdim : nullptr;
  const float* start = (LOCAL || only) ? S : B;
  const T* qsrc = proj + (size_t)h * dim;
  const T* vsrc = proj + 2 * (size_t)H * dim + (size_t)h * vdim + col0;
  const int cols_here = min(BC, vdim - col0);
  const bool wide = dim % 8 == 0 && vdim % 8 == 0 && ld % 8 == 0 && (((uintptr_t)proj | (uintptr_t)alpha) & 15) == 0;

  auto stage = [&](int ts, unsigned char* buf) {
    const int n = min(LA_STAGE, t1 - ts);
    if (wide) {
      constexpr int QP = RP / EPP, AP = RP / 4, VP = BC / EPP, PIECES = (LOCAL ? 1 : 2) * QP + AP + VP;
      for (int i = threadIdx.x; i < n * PIECES; i += blockDim.x) {
        const int tok = i / PIECES;
        int e = i - tok * PIECES;
        unsigned char* row = buf + tok * Z::BYTES;
        const T* src = qsrc + (size_t)(ts + tok) * ld;
        const void* from;
        unsigned char* to;
        bool there;
        if (e < QP) {
          there = e * EPP < dim;
          from = src + (size_t)H * dim + e * EPP;
          to = row + Z::K_AT + e * 16;
        } else if ((e -= QP) < AP) {
          there = e * 4 < dim;
          from = alpha + ((size_t)(ts + tok) * H + h) * dim + e * 4;
          to = row + Z::A_AT + e * 16;
        } else if ((e -= AP) < VP) {
          there = e * EPP < cols_here;
          from = vsrc + (size_t)(ts + tok) * ld + e * EPP;
          to = row + Z::V_AT + e * 16;
        } else {
          e -= VP;
          there = e * EPP < dim;
          from = src + e * EPP;
          to = row + e * 16;
        }
        if (there) la_copy16(to, from);
        else *reinterpret_cast<uint4*>(to) = make_uint4(0, 0, 0, 0);
      }
    } else {
      for (int i = threadIdx.x; i < n * (RP + BC); i += blockDim.x) {
        const int tok = i / (RP + BC), e = i - tok * (RP + BC);
        unsigned char* row = buf + tok * Z::BYTES;
        if (e < RP) {
          const T* src = qsrc + (size_t)(ts + tok) * ld + e;
          if (!LOCAL) reinterpret_cast<T*>(row)[e] = e < dim ? src[0] : from_float<T>(0.f);
          reinterpret_cast<T*>(row + Z::K_AT)[e] = e < dim ? src[(size_t)H * dim] : from_float<T>(0.f);
          reinterpret_cast<float*>(row + Z::A_AT)[e] = e < dim ? alpha[((size_t)(ts + tok) * H + h) * dim + e] : 0.f;
        } else {
          reinterpret_cast<T*>(row + Z::V_AT)[e - RP] = e - RP < cols_here ? vsrc[(size_t)(ts + tok) * ld + e - RP] : from_float<T>(0.f);
        }
      }
    }
    la_commit();
  };

  stage(t0, staged);
  const bool runs = NC == 4 && vdim % 4 == 0 && (((uintptr_t)start | (uintptr_t)S | (uintptr_t)B) & 15) == 0;
  float s[NC][PER], prod[PER];
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int d = row_of<PER, R>(r, e);
    prod[e] = 1.f;
#pragma unroll
    for (int j = 0; j < NC; ++j) s[j][e] = 0.f;
    if (!LOCAL && d < dim) {
      if (runs) {
        if (col < vdim) {
          const float4 v = *reinterpret_cast<const float4*>(start + (size_t)d * vdim + col);
          s[0][e] = v.x; s[1][e] = v.y; s[NC - 2][e] = v.z; s[NC - 1][e] = v.w;
        }
      } else {
#pragma unroll
        for (int j = 0; j < NC; ++j)
          if (col + j < vdim) s[j][e] = start[(size_t)d * vdim + col + j];
      }
    }
  }
  const bool with_products = LOCAL && blockIdx.x == 0 && warp == 0 && lane < R;
  int which = 0;
  for (int ts = t0; ts < t1; ts += LA_STAGE, which ^= 1) {
    const int n = min(LA_STAGE, t1 - ts);
    la_wait();
    __syncthreads();  // this stage has landed for everybody, and everybody has left the other buffer
    if (ts + LA_STAGE < t1) stage(ts + LA_STAGE, staged + (which ^ 1) * LA_STAGE * Z::BYTES);
    const unsigned char* buf = staged + which * LA_STAGE * Z::BYTES;
#pragma unroll 1
    for (int i = 0; i < n; ++i) {
      const unsigned char* row = buf + i * Z::BYTES;
      float kk[PER], aa[PER], v[NC];
      lane_vector<PER, R>(reinterpret_cast<const T*>(row + Z::K_AT), r, kk);
      lane_vector<PER, R>(reinterpret_cast<const float*>(row + Z::A_AT), r, aa);
#pragma unroll
      for (int j = 0; j < NC; ++j) v[j] = to_float<T>(reinterpret_cast<const T*>(row + Z::V_AT)[in_block + j]);
#pragma unroll
      for (int j = 0; j < NC; ++j)
#pragma unroll
        for (int e = 0; e < PER; ++e) s[j][e] = fmaf(kk[e], v[j], aa[e] * s[j][e]);
      if (LOCAL) {
        if (with_products) {
#pragma unroll
          for (int e = 0; e < PER; ++e) prod[e] *= aa[e];
        }
      } else {
        lane_vector<PER, R>(reinterpret_cast<const T*>(row), r, kk);
        float sum[NC];
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          float part[2] = {};
#pragma unroll
          for (int e = 0; e < PER; ++e) part[e & 1] = fmaf(kk[e], s[j][e], part[e & 1]);
          sum[j] = part[0] + part[1];
        }
        int mine = 0;  // which of the NC columns this lane ends up with
#pragma unroll
        for (int w = NC, off = 1; w > 1; w >>= 1, off <<= 1) {
          const bool up = r & off;
#pragma unroll
          for (int j = 0; j < w / 2; ++j) {
            const float give = up ? sum[j] : sum[j + w / 2], keep = up ? sum[j + w / 2] : sum[j];
            sum[j] = keep + __shfl_xor_sync(0xffffffffu, give, off);
          }
          mine += up ? w / 2 : 0;
        }
#pragma unroll
        for (int off = NC; off < R; off <<= 1) sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], off);
        if (r < NC && col + mine < vdim) o[((size_t)(ts + i) * H + h) * vdim + col + mine] = sum[0] * scale;
      }
    }
  }
  if (LOCAL || last) {
    float* dst = LOCAL ? B : S;
#pragma unroll
    for (int e = 0; e < PER; ++e) {
      const int d = row_of<PER, R>(r, e);
      if (d >= dim) continue;
      if (runs) {
        if (col < vdim) *reinterpret_cast<float4*>(dst + (size_t)d * vdim + col) = make_float4(s[0][e], s[1][e], s[NC - 2][e], s[NC - 1][e]);
      } else {
#pragma unroll
        for (int j = 0; j < NC; ++j)
          if (col + j < vdim) dst[(size_t)d * vdim + col + j] = s[j][e];
      }
    }
  }
  if (with_products) {
    float* A = local_a + ((size_t)blockIdx.z * H + h) * dim;
#pragma unroll
    for (int e = 0; e < PER; ++e) {
      const int d = row_of<PER, R>(r, e);
      if (d < dim) A[d] = prod[e];
    }
  }
}

// A thread per number of a portion's state: B of every chunk becomes the state the chunk starts from.
__global__ void __launch_bounds__(256)
linear_attention_starts_kernel(const float* __restrict__ state, long long slot_floats, const int32_t* __restrict__ item_start,
                               const int32_t* __restrict__ slots, float* __restrict__ local_b, const float* __restrict__ local_a,
                               int H, int dim, int vdim, int num_slots, int chunk) {
  pdl_trigger();
  pdl_wait();
  const int item = blockIdx.y;
  int first = 0;
  for (int i = 0; i < item; ++i) first += (item_start[i + 1] - item_start[i] + chunk - 1) / chunk;
  const int n = (item_start[item + 1] - item_start[item] + chunk - 1) / chunk;
  const long long per_chunk = (long long)H * dim * vdim;
  const long long at = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (n <= 1 || at >= per_chunk) return;
  int slot = slots[item];
  slot = slot < 0 ? 0 : (slot >= num_slots ? num_slots - 1 : slot);
  float run = state[(size_t)slot * slot_floats + at];
  const long long hd = at / vdim;
  constexpr int AHEAD = 8;
  for (int c0 = 0; c0 < n; c0 += AHEAD) {
    float b[AHEAD], a[AHEAD];
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {  // asked for together; the last chunk has neither
      const int c = c0 + j;
      b[j] = c < n - 1 ? local_b[(size_t)(first + c) * per_chunk + at] : 0.f;
      a[j] = c < n - 1 ? local_a[(size_t)(first + c) * H * dim + hd] : 0.f;
    }
#pragma unroll
    for (int j = 0; j < AHEAD; ++j) {
      const int c = c0 + j;
      if (c >= n) break;
      local_b[(size_t)(first + c) * per_chunk + at] = run;
      run = fmaf(a[j], run, b[j]);
    }
  }
}

enum : int { READOUT_GATE_PLAIN = 0, READOUT_GATE_SILU = 1, READOUT_GATE_SIGMOID = 2 };

template <typename TG, typename TO>
__global__ void __launch_bounds__(128)
normed_readout_kernel(const float* __restrict__ o, const TG* __restrict__ gate, long long ldg, int gate_act,
                      const float* __restrict__ gain, int head_gains, TO* __restrict__ out, long long ldo, long long units, int H,
                      int vdim, float eps) {
  pdl_trigger();
  pdl_wait();
  const long long unit = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (unit >= units) return;
  const long long t = unit / H;
  const int h = (int)(unit - t * H);
  const float* row = o + (size_t)unit * vdim;
  const TG* g = gate + (size_t)t * ldg + (size_t)h * vdim;
  float ss = 0.f;
  for (int j = lane; j < vdim; j += 32) ss = fmaf(row[j], row[j], ss);
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)vdim + eps);
  TO* dst = out + (size_t)t * ldo + (size_t)h * vdim;
  if (head_gains) gain += (size_t)h * vdim;
  for (int j = lane; j < vdim; j += 32) {
    float v = to_float<TG>(g[j]);
    if (gate_act == READOUT_GATE_SILU) v = v / (1.f + expf(-v));
    else if (gate_act == READOUT_GATE_SIGMOID) v = 1.f / (1.f + expf(-v));
    dst[j] = from_float<TO>(row[j] * inv * gain[j] * v);
  }
}

}  // namespace

// (proj, dtype, ld, alpha, state, slot_floats, item_start, slots, local_b, local_a, o, items, chunks, H, dim, vdim, num_slots,
//  chunk, scale, stream).  ``chunks``: blocks to launch, at least the number of chunks of the step's portions; local_b
// [chunks, H, dim, vdim] and local_a [chunks, H, dim] float32 are scratch, null when no portion is longer than a chunk.
PSB_API int psb_linear_attention(const void* proj, int dtype, long long ld, const void* alpha, void* state, long long slot_floats,
                                 const void* item_start, const void* slots, void* local_b, void* local_a, void* o, int items,
                                 int chunks, int H, int dim, int vdim, int num_slots, int chunk, float scale, cudaStream_t stream) {
  if (items < 0 || H < 1 || dim < 1 || vdim < 1 || chunk < 1 || num_slots < 1) PSB_REFUSE("linear_attention: bad sizes H=%d dim=%d vdim=%d", H, dim, vdim);
  if (ld < 2LL * H * dim + (long long)H * vdim) PSB_REFUSE("linear_attention: row stride %lld is shorter than the row", ld);
  if (slot_floats < (long long)H * dim * vdim) PSB_REFUSE("linear_attention: a slot of %lld numbers does not hold the state", slot_floats);
  if (dim > 1024) PSB_REFUSE("linear_attention: key size %d exceeds 1024", dim);
  if ((local_a == nullptr) != (local_b == nullptr)) PSB_REFUSE("linear_attention: the two scratch arrays come together");
  if (H > 65535 || chunks > 65535 || items > 65535 || chunks < items) PSB_REFUSE("linear_attention: too many heads, requests or chunks for one launch");
  if (items == 0) return 0;
#define PSB_LA(PER_, R_, NC_)                                                                                                    \
  do {                                                                                                                           \
    using Z = LaSizes<T, PER_, R_, NC_>;                                                                                          \
    constexpr size_t smem = Z::SMEM;                                                                                              \
    const dim3 grid((vdim + Z::BC - 1) / Z::BC, H, chunks);                                                                       \
    auto local = linear_attention_kernel<T, PER_, R_, NC_, true>;                                                                 \
    auto whole = linear_attention_kernel<T, PER_, R_, NC_, false>;                                                                \
    if (smem > 48 * 1024) {                                                                                                       \
      static PsbPerDevice configured;                                                                                             \
      if (!configured.get()) {                                                                                                    \
        if (cudaFuncSetAttribute(local, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess ||                 \
            cudaFuncSetAttribute(whole, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)                   \
          PSB_REFUSE("linear_attention: cannot raise the shared-memory limit");                                                   \
        configured.set();                                                                                                         \
      }                                                                                                                           \
    }                                                                                                                             \
    if (local_b) {                                                                                                                \
      psb_launch(local, grid, dim3(LA_WARPS * 32), smem, stream, (const T*)proj, ld, (const float*)alpha, (float*)state,          \
                 slot_floats, (const int32_t*)item_start, (const int32_t*)slots, (float*)local_b, (float*)local_a, (float*)o,     \
                 items, H, dim, vdim, num_slots, chunk, scale);                                                                   \
      PSB_LAUNCH_CHECK("linear_attention");                                                                                       \
      const long long per = (long long)H * dim * vdim;                                                                            \
      psb_launch(linear_attention_starts_kernel, dim3((unsigned)((per + 255) / 256), items), dim3(256), 0, stream,                \
                 (const float*)state, slot_floats, (const int32_t*)item_start, (const int32_t*)slots, (float*)local_b,            \
                 (const float*)local_a, H, dim, vdim, num_slots, chunk);                                                          \
      PSB_LAUNCH_CHECK("linear_attention_starts");                                                                                \
    }                                                                                                                             \
    psb_launch(whole, grid, dim3(LA_WARPS * 32), smem, stream, (const T*)proj, ld, (const float*)alpha, (float*)state,            \
               slot_floats, (const int32_t*)item_start, (const int32_t*)slots, (float*)local_b, (float*)local_a, (float*)o,       \
               items, H, dim, vdim, num_slots, chunk, scale);                                                                     \
    PSB_LAUNCH_CHECK("linear_attention");                                                                                         \
  } while (0)
  PSB_DISPATCH_DTYPE(dtype, T, {
    if (dim <= 16) PSB_LA(4, 4, 4);
    else if (dim <= 32) PSB_LA(8, 4, 4);
    else if (dim <= 64) PSB_LA(8, 8, 4);
    else if (dim <= 128) PSB_LA(16, 8, 4);
    else if (dim <= 256) PSB_LA(16, 16, 4);
    else if (dim <= 512) PSB_LA(16, 32, 4);
    else PSB_LA(32, 32, 2);
  });
#undef PSB_LA
  return 0;
}

// (o float32 [T, H, vdim], gate, gate_dtype, ldg, gate_act, gain [vdim] or with head_gains [H, vdim], head_gains, out in rows ldo
// numbers apart, out_dtype, ldo, T, H, vdim, eps, stream)
PSB_API int psb_normed_readout(const void* o, const void* gate, int gate_dtype, long long ldg, int gate_act, const void* gain,
                               int head_gains, void* out, int out_dtype, long long ldo, int T, int H, int vdim, float eps,
                               cudaStream_t stream) {
  if (T < 0 || H < 1 || vdim < 1 || ldg < (long long)H * vdim || ldo < (long long)H * vdim)
    PSB_REFUSE("normed_readout: bad sizes H=%d vdim=%d ldg=%lld ldo=%lld", H, vdim, ldg, ldo);
  if (gate_act != READOUT_GATE_PLAIN && gate_act != READOUT_GATE_SILU && gate_act != READOUT_GATE_SIGMOID) PSB_REFUSE("normed_readout: gate code %d is not built", gate_act);
  if (T == 0) return 0;
  const long long units = (long long)T * H;
  PSB_DISPATCH_DTYPE(gate_dtype, TG, {
    PSB_DISPATCH_DTYPE(out_dtype, TO, {
      psb_launch(normed_readout_kernel<TG, TO>, dim3((unsigned)((units + 3) / 4)), dim3(128), 0, stream, (const float*)o,
                 (const TG*)gate, ldg, gate_act, (const float*)gain, head_gains, (TO*)out, ldo, units, H, vdim, eps);
    });
  });
  PSB_LAUNCH_CHECK("normed_readout");
  return 0;
}

// What lies between the fused projection of an attention layer and its scores, for designs that do more to queries
// and keys than rotate them: per token, in one pass over the projection's row [q | k | v] (or [q | k] where the
// projected keys serve as values),
//
//   rotation of the first ``rotary_dim`` elements of every query and key head by the token's absolute position
//     (optional; ``interleaved``: element 2i turns with 2i+1, else i with i + rotary_dim/2);
//   division of every query and key head by the root of (its mean square + eps)   (optional: eps < 0 leaves it out);
//   a factor per query head (optional), so that a head's scores come out multiplied by it;
//   the query written to q_out [T, hq, dim]; the key, then the value, to the token's row of the cache entry
//     [num_pages, 1, hkv, page_size, dim + vdim], the value being the head's own projection or, with
//     ``values_are_keys``, the key as it was projected (before rotation and norm).  With ``split_planes`` (vdim == dim)
//     the entry is [num_pages, 2, hkv, page_size, dim] instead, keys in plane 0 and values in plane 1: the layout of
//     the attention kernels that read keys and values as separate tiles.
//
// Two kernels.  The general one: one block per token, a warp per head in turn; the head lies in the warp's
// shared-memory row between the steps.  The other, for heads of 64, 128 or 256 elements whose rotation (if any) pairs
// neighbours: the head in registers, 32 or 16 lanes a head (every lane a run of elements, which holds whole pairs), one
// wide load and one wide store per lane and row, a warp taking one or several heads.
// Rotation, statistics and factors are float32; storage is float32 or bfloat16.
//
// attention_prepare_heads_*: the pass of layers whose query and key heads are each RMS-normed with a gain over the head's
// elements (one for all query heads, one for all key heads) before the rotation, and whose values may be mixed with those of
// an earlier layer: v <- (1 - share) v + share * first.  Biases come first, in float32.
#include "common.cuh"

namespace {

constexpr int PREP_WARPS = 4;
constexpr int PREP_MAX_D = 256;

template <typename T, typename TKV>
__global__ void __launch_bounds__(PREP_WARPS * 32)
attention_prepare_kernel(const T* __restrict__ proj, long long ld, const int32_t* __restrict__ positions,
                         const int32_t* __restrict__ token_item, const int32_t* __restrict__ table, int table_width,
                         const float* __restrict__ cos_t, const float* __restrict__ sin_t, const float* __restrict__ head_factor,
                         TKV* __restrict__ kv, T* __restrict__ q_out, int hq, int hkv, int dim, int vdim, int page_size,
                         int num_pages, int max_positions, int rotary_dim, int interleaved, float eps, int values_are_keys,
                         int split_planes, const float* __restrict__ bias, int write_kv) {
  __shared__ float rows[PREP_WARPS][PREP_MAX_D];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qw = hq * dim, kw = hkv * dim;
  const T* row = proj + (size_t)t * ld;  // ld >= the row's width: the projection may be a run of columns of a wider product
  const int p = positions[t];
  const int page = write_kv ? table[(size_t)token_item[t] * table_width + p / page_size] : -1;
  const bool page_ok = page >= 0 && page < num_pages;  // tables are checked on the host; never write outside the pool
  const int rw = dim + vdim;
  const int half = rotary_dim / 2;
  const bool turn = cos_t != nullptr && p >= 0 && p < max_positions;
  const float* cs = turn ? cos_t + (size_t)p * half : nullptr;
  const float* sn = turn ? sin_t + (size_t)p * half : nullptr;
  float* mine = rows[warp];
  // ``bias`` (float32, one number per column of the row, optional) is added to the projection in float32;
  // ``write_kv`` 0: the row holds queries only (a layer that reads another layer's keys and values)
  for (int head = warp; head < hq + (write_kv ? hkv : 0); head += PREP_WARPS) {
    const bool is_q = head < hq;
    const T* src = row + (size_t)head * dim;  // query heads, then key heads, lie one after the other
    for (int d = lane; d < dim; d += 32) mine[d] = to_float<T>(src[d]) + (bias ? bias[(size_t)head * dim + d] : 0.f);
    __syncwarp();
    if (turn) {
      for (int i = lane; i < half; i += 32) {
        const int a = interleaved ? 2 * i : i, b = interleaved ? 2 * i + 1 : i + half;
        float o1, o2;
        rotate_pair(mine[a], mine[b], cs[i], sn[i], o1, o2);
        mine[a] = o1;
        mine[b] = o2;
      }
      __syncwarp();
    }
    float factor = 1.f;
    if (eps >= 0.f) {
      float ss = 0.f;
      for (int d = lane; d < dim; d += 32) ss = fmaf(mine[d], mine[d], ss);
      factor = 1.f / sqrtf(warp_sum(ss) / (float)dim + eps);
    }
    if (is_q) {
      const float f = head_factor ? head_factor[head] : 1.f;
      T* dst = q_out + ((size_t)t * hq + head) * dim;
      for (int d = lane; d < dim; d += 32) dst[d] = from_float<T>(mine[d] * factor * f);
    } else if (page_ok) {
      const int g = head - hq;
      const size_t slot = (size_t)(p % page_size);
      TKV* dst = split_planes ? kv + ((((size_t)page * 2) * hkv + g) * page_size + slot) * dim
                              : kv + (((size_t)page * hkv + g) * page_size + slot) * rw;
      TKV* vdst = split_planes ? dst + (size_t)hkv * page_size * dim : dst + dim;
      for (int d = lane; d < dim; d += 32) dst[d] = from_float<TKV>(mine[d] * factor);
      const T* vsrc = values_are_keys ? src : row + qw + kw + (size_t)g * vdim;
      const float* vb = bias ? (values_are_keys ? bias + (size_t)head * dim : bias + qw + kw + (size_t)g * vdim) : nullptr;
      for (int d = lane; d < vdim; d += 32) vdst[d] = from_float<TKV>(to_float<T>(vsrc[d]) + (vb ? vb[d] : 0.f));
    }
    __syncwarp();
  }
}

// A run of N elements that is loaded and stored as one piece.
template <typename T, int N>
struct alignas(sizeof(T) * N) Run {
  T v[N];
};

// grid: T * groups blocks.  LPH lanes hold a head (32, or 16 for heads of 64 when both head counts are even: then a lane has
// four elements instead of two and a warp takes two heads at a time, which halves the instructions a byte costs); a warp
// takes HPW rounds of 32 / LPH heads: heads (warp index in the token * HPW + round) * (32 / LPH) + lane / LPH.  HPW > 1 (long
// steps): the rows of all of a warp's rounds are asked for together, before any of them is used, so that a lane has
// several loads in flight.  groups = ceil((hq + hkv) / (PREP_WARPS * HPW * 32 / LPH)).  A round lies within the heads or
// beyond them as a whole (the head counts are multiples of 32 / LPH), so the shuffles of a round see all of its lanes.
template <typename T, typename TKV, int DIM, int HPW, int LPH>
__global__ void __launch_bounds__(PREP_WARPS * 32)
attention_prepare_rows_kernel(const T* __restrict__ proj, long long ld, const int32_t* __restrict__ positions,
                              const int32_t* __restrict__ token_item, const int32_t* __restrict__ table, int table_width,
                              const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                              const float* __restrict__ head_factor, TKV* __restrict__ kv, T* __restrict__ q_out, int hq, int hkv,
                              int page_size, int num_pages, int max_positions, int rotary_dim, float eps, int values_are_keys,
                              int split_planes, int groups) {
  constexpr int N = DIM / LPH;    // elements a lane holds
  constexpr int HPR = 32 / LPH;   // heads a round
  pdl_trigger();
  const int t = blockIdx.x / groups;
  const int lane = threadIdx.x & 31;
  const int sub = lane / LPH, sl = lane % LPH;
  const int head0 = ((blockIdx.x - t * groups) * PREP_WARPS + (threadIdx.x >> 5)) * HPW * HPR;
  // positions and tables are inputs of the step: they may be read before the preceding kernel has finished
  const int p = positions[t];
  const int page = table[(size_t)token_item[t] * table_width + p / page_size];
  pdl_wait();
  const int heads = hq + hkv;
  if (head0 >= heads) return;
  const T* row = proj + (size_t)t * ld;
  Run<T, N> raw[HPW], vin[HPW];
#pragma unroll
  for (int i = 0; i < HPW; ++i) {
    const int head = head0 + i * HPR + sub;
    if (head < heads) raw[i] = *reinterpret_cast<const Run<T, N>*>(row + (size_t)head * DIM + sl * N);
    if (head < heads && head >= hq && !values_are_keys)
      vin[i] = *reinterpret_cast<const Run<T, N>*>(row + (size_t)heads * DIM + (size_t)(head - hq) * DIM + sl * N);
  }
  const bool turn = cos_t != nullptr && p >= 0 && p < max_positions;
  float cs[N / 2], sn[N / 2];
  if (turn) {
#pragma unroll
    for (int i = 0; i < N; i += 2) {
      const int d = sl * N + i;  // even: the pair (d, d + 1) turns by angle d / 2
      cs[i / 2] = d < rotary_dim ? cos_t[(size_t)p * (rotary_dim / 2) + (d >> 1)] : 1.f;
      sn[i / 2] = d < rotary_dim ? sin_t[(size_t)p * (rotary_dim / 2) + (d >> 1)] : 0.f;
    }
  }
#pragma unroll
  for (int hh = 0; hh < HPW; ++hh) {
    const int head = head0 + hh * HPR + sub;
    if (head0 + hh * HPR >= heads) break;  // the whole round lies beyond the heads
    float x[N];
#pragma unroll
    for (int i = 0; i < N; ++i) x[i] = to_float<T>(raw[hh].v[i]);
    if (turn) {
#pragma unroll
      for (int i = 0; i < N; i += 2) {
        if (sl * N + i < rotary_dim) {
          float o1, o2;
          rotate_pair(x[i], x[i + 1], cs[i / 2], sn[i / 2], o1, o2);
          x[i] = o1;
          x[i + 1] = o2;
        }
      }
    }
    float factor = 1.f;
    if (eps >= 0.f) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < N; ++i) ss = fmaf(x[i], x[i], ss);
#pragma unroll
      for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);  // over the head's lanes
      factor = 1.f / sqrtf(ss / (float)DIM + eps);
    }
    if (head >= heads) continue;  // cannot happen while the head counts are multiples of a round; never store for a head that is not there
    if (head < hq) {
      const float f = head_factor ? head_factor[head] : 1.f;
      Run<T, N> o;
#pragma unroll
      for (int i = 0; i < N; ++i) o.v[i] = from_float<T>(x[i] * factor * f);
      *reinterpret_cast<Run<T, N>*>(q_out + ((size_t)t * hq + head) * DIM + sl * N) = o;
      continue;
    }
    if (page < 0 || page >= num_pages) continue;  // tables are checked on the host; never write outside the pool
    const int g = head - hq;
    const size_t slot = (size_t)(p % page_size);
    TKV* dst = split_planes ? kv + ((((size_t)page * 2) * hkv + g) * page_size + slot) * DIM
                            : kv + (((size_t)page * hkv + g) * page_size + slot) * (2 * DIM);
    TKV* vdst = split_planes ? dst + (size_t)hkv * page_size * DIM : dst + DIM;
    Run<TKV, N> k;
#pragma unroll
    for (int i = 0; i < N; ++i) k.v[i] = from_float<TKV>(x[i] * factor);
    *reinterpret_cast<Run<TKV, N>*>(dst + sl * N) = k;
    const Run<T, N> vsrc = values_are_keys ? raw[hh] : vin[hh];
    Run<TKV, N> v;
#pragma unroll
    for (int i = 0; i < N; ++i) v.v[i] = from_float<TKV>(to_float<T>(vsrc.v[i]));
    *reinterpret_cast<Run<TKV, N>*>(vdst + sl * N) = v;
  }
}

// The pass of attention layers whose whole query projection and whole key projection (all heads at once) are each RMS-normed
// with a gain per column, after their biases and without a rotation: a block per token, the row's columns in runs of N (N
// divides the head sizes; 8 where the addresses allow), float32 in between.  Cache entry and layouts as above.
template <typename T, typename TKV, int N>
__global__ void __launch_bounds__(256)
attention_prepare_normed_kernel(const T* __restrict__ proj, long long ld, const int32_t* __restrict__ positions,
                                const int32_t* __restrict__ token_item, const int32_t* __restrict__ table, int table_width,
                                const float* __restrict__ bias, const float* __restrict__ gain, TKV* __restrict__ kv,
                                T* __restrict__ q_out, int hq, int hkv, int dim, int vdim, int page_size, int num_pages, float eps,
                                int split_planes) {
  __shared__ float2 scratch[8];
  constexpr int KEEP = N == 8 ? 4 : 1;  // runs a thread keeps from the first pass to the second (later ones are read again)
  pdl_trigger();
  const int t = blockIdx.x;
  const int p = positions[t];  // inputs of the step: they may be read before the preceding kernel has finished
  const int page = table[(size_t)token_item[t] * table_width + p / page_size];
  pdl_wait();
  const int qw = hq * dim, kw = hkv * dim, vw = hkv * vdim;
  const T* row = proj + (size_t)t * ld;
  float sq = 0.f, sk = 0.f;
  auto biased = [&](int c, float (&x)[N]) {
    const Run<T, N> raw = *reinterpret_cast<const Run<T, N>*>(row + c);
    Run<float, N> b = {};
    if (bias) b = *reinterpret_cast<const Run<float, N>*>(bias + c);
#pragma unroll
    for (int i = 0; i < N; ++i) x[i] = to_float<T>(raw.v[i]) + b.v[i];
  };
  auto add = [&](int c, const float (&x)[N]) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) ss = fmaf(x[i], x[i], ss);
    if (c < qw) sq += ss;
    else if (c < qw + kw) sk += ss;
  };
  float held[KEEP][N];
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = (k * blockDim.x + threadIdx.x) * N;
    if (c < qw + kw + vw) biased(c, held[k]);
  }
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = (k * blockDim.x + threadIdx.x) * N;
    if (c < qw + kw) add(c, held[k]);
  }
  for (int c = (KEEP * blockDim.x + threadIdx.x) * N; c < qw + kw; c += blockDim.x * N) {
    float x[N];
    biased(c, x);
    add(c, x);
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((threadIdx.x & 31) == 0) scratch[threadIdx.x >> 5] = make_float2(sq, sk);
  __syncthreads();
  sq = sk = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) {
    sq += scratch[w].x;
    sk += scratch[w].y;
  }
  const float iq = 1.f / sqrtf(sq / (float)qw + eps), ik = 1.f / sqrtf(sk / (float)kw + eps);
  const bool page_ok = page >= 0 && page < num_pages;  // tables are checked on the host; never write outside the pool
  const size_t slot = (size_t)(p % page_size);
  auto put = [&](int c, const float (&x)[N]) {
    Run<float, N> g = {};
    if (c < qw + kw) g = *reinterpret_cast<const Run<float, N>*>(gain + c);
    if (c < qw) {
      Run<T, N> o;
#pragma unroll
      for (int i = 0; i < N; ++i) o.v[i] = from_float<T>(g.v[i] * (x[i] * iq));
      *reinterpret_cast<Run<T, N>*>(q_out + (size_t)t * qw + c) = o;
      return;
    }
    if (!page_ok) return;
    Run<TKV, N> o;
    TKV* dst;
    if (c < qw + kw) {
      const int head = (c - qw) / dim, d = (c - qw) - head * dim;
#pragma unroll
      for (int i = 0; i < N; ++i) o.v[i] = from_float<TKV>(g.v[i] * (x[i] * ik));
      dst = split_planes ? kv + ((((size_t)page * 2) * hkv + head) * page_size + slot) * dim + d
                         : kv + (((size_t)page * hkv + head) * page_size + slot) * (dim + vdim) + d;
    } else {
      const int head = (c - qw - kw) / vdim, d = (c - qw - kw) - head * vdim;
#pragma unroll
      for (int i = 0; i < N; ++i) o.v[i] = from_float<TKV>(x[i]);
      dst = split_planes ? kv + ((((size_t)page * 2 + 1) * hkv + head) * page_size + slot) * dim + d
                         : kv + (((size_t)page * hkv + head) * page_size + slot) * (dim + vdim) + dim + d;
    }
    *reinterpret_cast<Run<TKV, N>*>(dst) = o;
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int c = (k * blockDim.x + threadIdx.x) * N;
    if (c < qw + kw + vw) put(c, held[k]);
  }
  for (int c = (KEEP * blockDim.x + threadIdx.x) * N; c < qw + kw + vw; c += blockDim.x * N) {
    float x[N];
    biased(c, x);
    put(c, x);
  }
}

// What the pass of layers with normed heads reads besides the projection.
template <typename T>
struct HeadsArgs {
  const T* proj;
  long long ld;
  const int32_t *positions, *token_item, *table;
  int table_width;
  const float *cos_t, *sin_t;             // [max_positions, rotary_dim / 2], null: no rotation
  const float* bias;                      // one number per column of [q | k | v], or null
  const float *gain_q, *gain_k;           // [dim] each
  const T* first;                         // an earlier layer's projected values of the same tokens (rows ld_first apart), or null
  long long ld_first;
  const float* first_bias;                // their biases [hkv * vdim], or null
  const float* share;                     // one number: the weight of ``first``
  T* q_out;                               // [T, hq, dim]
  int tokens, hq, hkv, dim, vdim, page_size, num_pages, max_positions, rotary_dim, interleaved, split_planes;
  float eps;
};

template <typename T, typename TKV>
__device__ __forceinline__ TKV* heads_row(const HeadsArgs<T>& a, TKV* kv, int page, int p, int g, bool value) {
  const size_t slot = (size_t)(p % a.page_size);
  if (a.split_planes) return kv + ((((size_t)page * 2 + (value ? 1 : 0)) * a.hkv + g) * a.page_size + slot) * a.dim;
  return kv + (((size_t)page * a.hkv + g) * a.page_size + slot) * (a.dim + a.vdim) + (value ? a.dim : 0);
}

// Any sizes: a block per token, a warp per head in turn, the head in the warp's shared-memory row between the steps.
template <typename T, typename TKV>
__global__ void __launch_bounds__(PREP_WARPS * 32)
attention_prepare_heads_kernel(const HeadsArgs<T> a, TKV* __restrict__ kv) {
  __shared__ float rows[PREP_WARPS][PREP_MAX_D];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qw = a.hq * a.dim, kw = a.hkv * a.dim, vw = a.hkv * a.vdim;
  const T* row = a.proj + (size_t)t * a.ld;
  const int p = a.positions[t];
  const int page = a.table[(size_t)a.token_item[t] * a.table_width + p / a.page_size];
  const bool page_ok = page >= 0 && page < a.num_pages;  // tables are checked on the host; never write outside the pool
  const int half = a.rotary_dim / 2;
  const bool turn = a.cos_t != nullptr && p >= 0 && p < a.max_positions;
  float* mine = rows[warp];
  for (int head = warp; head < a.hq + a.hkv; head += PREP_WARPS) {
    const bool is_q = head < a.hq;
    float ss = 0.f;
    for (int d = lane; d < a.dim; d += 32) {
      const int c = head * a.dim + d;
      const float x = to_float<T>(row[c]) + (a.bias ? a.bias[c] : 0.f);
      mine[d] = x;
      ss = fmaf(x, x, ss);
    }
    const float factor = 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
    const float* gain = is_q ? a.gain_q : a.gain_k;
    for (int d = lane; d < a.dim; d += 32) mine[d] = mine[d] * factor * gain[d];
    __syncwarp();
    if (turn) {
      for (int i = lane; i < half; i += 32) {
        const int lo = a.interleaved ? 2 * i : i, hi = a.interleaved ? 2 * i + 1 : i + half;
        float o1, o2;
        rotate_pair(mine[lo], mine[hi], a.cos_t[(size_t)p * half + i], a.sin_t[(size_t)p * half + i], o1, o2);
        mine[lo] = o1;
        mine[hi] = o2;
      }
      __syncwarp();
    }
    if (is_q) {
      for (int d = lane; d < a.dim; d += 32) a.q_out[((size_t)t * a.hq + head) * a.dim + d] = from_float<T>(mine[d]);
    } else if (page_ok) {
      TKV* dst = heads_row<T, TKV>(a, kv, page, p, head - a.hq, false);
      for (int d = lane; d < a.dim; d += 32) dst[d] = from_float<TKV>(mine[d]);
    }
    __syncwarp();
  }
  if (!page_ok) return;
  const float share = a.first ? *a.share : 0.f;
  for (int c = threadIdx.x; c < vw; c += blockDim.x) {
    float v = to_float<T>(row[qw + kw + c]) + (a.bias ? a.bias[qw + kw + c] : 0.f);
    if (a.first) v = (1.f - share) * v + share * (to_float<T>(a.first[(size_t)t * a.ld_first + c]) + (a.first_bias ? a.first_bias[c] : 0.f));
    const int g = c / a.vdim;
    heads_row<T, TKV>(a, kv, page, p, g, true)[c - g * a.vdim] = from_float<TKV>(v);
  }
}

// Heads of 8 * LPH elements in registers: a thread takes the same run of eight columns of TOK tokens (bias and gains are
// fetched once, the tokens' loads are in flight together), LPH lanes a head.  Threads 0 .. heads * LPH - 1 (rounded up to whole
// warps) hold query and key heads, the ones behind them values.  A rotation of halves finds its partner 8 columns times a power
// of two away, one exchange between two lanes.
template <typename T, typename TKV, int LPH, int TOK>
__global__ void __launch_bounds__(256)
attention_prepare_heads_vec_kernel(const HeadsArgs<T> a, TKV* __restrict__ kv) {
  pdl_trigger();
  const int heads = a.hq + a.hkv, dim = 8 * LPH;
  const int head_threads = (heads * LPH + 31) & ~31;
  const int at = blockIdx.y * blockDim.x + threadIdx.x;
  const bool is_value = at >= head_threads;
  const int vrun = at - head_threads;
  const bool there = is_value ? vrun * 8 < a.hkv * a.vdim : at < heads * LPH;
  const int col = is_value ? heads * dim + vrun * 8 : at * 8;
  const int t0 = blockIdx.x * TOK;
  int pos[TOK], page[TOK];
#pragma unroll
  for (int k = 0; k < TOK; ++k) {  // inputs of the step: they may be read before the preceding kernel has finished
    const int t = min(t0 + k, a.tokens - 1);
    pos[k] = a.positions[t];
    page[k] = a.table[(size_t)a.token_item[t] * a.table_width + pos[k] / a.page_size];
    if (page[k] >= a.num_pages) page[k] = -1;  // tables are checked on the host; never write outside the pool
  }
  Run<float, 8> b = {}, g = {};
  if (there) {
    if (a.bias) b = *reinterpret_cast<const Run<float, 8>*>(a.bias + col);
    if (!is_value) g = *reinterpret_cast<const Run<float, 8>*>((at / LPH < a.hq ? a.gain_q : a.gain_k) + (at % LPH) * 8);
  }
  pdl_wait();
  Run<T, 8> raw[TOK], first[TOK];
#pragma unroll
  for (int k = 0; k < TOK; ++k) {
    raw[k] = first[k] = Run<T, 8>{};
    if (there && t0 + k < a.tokens) {
      raw[k] = *reinterpret_cast<const Run<T, 8>*>(a.proj + (size_t)(t0 + k) * a.ld + col);
      if (is_value && a.first) first[k] = *reinterpret_cast<const Run<T, 8>*>(a.first + (size_t)(t0 + k) * a.ld_first + vrun * 8);
    }
  }
  if (is_value) {
    if (!there) return;
    const int head = vrun * 8 / a.vdim, d = vrun * 8 - head * a.vdim;
    Run<float, 8> fb = {};
    if (a.first && a.first_bias) fb = *reinterpret_cast<const Run<float, 8>*>(a.first_bias + vrun * 8);
    const float share = a.first ? *a.share : 0.f;
#pragma unroll
    for (int k = 0; k < TOK; ++k) {
      if (t0 + k >= a.tokens || page[k] < 0) continue;
      Run<TKV, 8> o;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        float v = to_float<T>(raw[k].v[i]) + b.v[i];
        if (a.first) v = (1.f - share) * v + share * (to_float<T>(first[k].v[i]) + fb.v[i]);
        o.v[i] = from_float<TKV>(v);
      }
      *reinterpret_cast<Run<TKV, 8>*>(heads_row<T, TKV>(a, kv, page[k], pos[k], head, true) + d) = o;
    }
    return;
  }
  const int sl = at % LPH, head = at / LPH, half = a.rotary_dim / 2;
#pragma unroll
  for (int k = 0; k < TOK; ++k) {
    float x[8];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      x[i] = to_float<T>(raw[k].v[i]) + b.v[i];
      ss = fmaf(x[i], x[i], ss);
    }
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);  // over the head's lanes
    const float factor = 1.f / sqrtf(ss / (float)dim + a.eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] = x[i] * factor * g.v[i];
    if (a.cos_t) {  // the same for every lane
      const int p = min(max(pos[k], 0), a.max_positions - 1);  // (a position beyond the tables is refused on the host)
      const float *cs = a.cos_t + (size_t)p * half, *sn = a.sin_t + (size_t)p * half;
      if (a.interleaved) {
#pragma unroll
        for (int i = 0; i < 8; i += 2) {
          const int d = sl * 8 + i;
          if (d >= a.rotary_dim) continue;
          float o1, o2;
          rotate_pair(x[i], x[i + 1], cs[d / 2], sn[d / 2], o1, o2);
          x[i] = o1;
          x[i + 1] = o2;
        }
      } else {
        const bool turns = sl * 8 < a.rotary_dim, upper = sl * 8 >= half;
        Run<float, 8> c = {}, s = {};
        if (turns) {
          c = *reinterpret_cast<const Run<float, 8>*>(cs + sl * 8 - (upper ? half : 0));
          s = *reinterpret_cast<const Run<float, 8>*>(sn + sl * 8 - (upper ? half : 0));
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float other = __shfl_xor_sync(0xffffffffu, x[i], half / 8);
          float o1, o2;
          rotate_pair(upper ? other : x[i], upper ? x[i] : other, c.v[i], s.v[i], o1, o2);
          if (turns) x[i] = upper ? o2 : o1;
        }
      }
    }
    if (!there || t0 + k >= a.tokens) continue;
    if (head < a.hq) {
      Run<T, 8> o;
#pragma unroll
      for (int i = 0; i < 8; ++i) o.v[i] = from_float<T>(x[i]);
      *reinterpret_cast<Run<T, 8>*>(a.q_out + ((size_t)(t0 + k) * a.hq + head) * dim + sl * 8) = o;
    } else if (page[k] >= 0) {
      Run<TKV, 8> o;
#pragma unroll
      for (int i = 0; i < 8; ++i) o.v[i] = from_float<TKV>(x[i]);
      *reinterpret_cast<Run<TKV, 8>*>(heads_row<T, TKV>(a, kv, page[k], pos[k], head - a.hq, false) + sl * 8) = o;
    }
  }
}

template <typename T, typename TKV, int LPH>
void launch_heads_vec(const HeadsArgs<T>& a, TKV* kv, cudaStream_t stream) {
  const int lanes = (((a.hq + a.hkv) * LPH + 31) & ~31) + ((a.hkv * (a.vdim / 8) + 31) & ~31);
  const int threads = lanes < 256 ? lanes : 256;
  const int tok = a.tokens >= 512 ? 2 : 1;
  const dim3 grid((a.tokens + tok - 1) / tok, (lanes + threads - 1) / threads);
  if (tok == 2) psb_launch(attention_prepare_heads_vec_kernel<T, TKV, LPH, 2>, grid, dim3(threads), 0, stream, a, kv);
  else psb_launch(attention_prepare_heads_vec_kernel<T, TKV, LPH, 1>, grid, dim3(threads), 0, stream, a, kv);
}

template <typename T, typename TKV>
void launch_heads(const HeadsArgs<T>& a, TKV* kv, cudaStream_t stream) {
  const int half8 = a.rotary_dim / 16;
  const uintptr_t in_run = 8 * sizeof(T), kv_run = 8 * sizeof(TKV);
  const bool turn_fits = !a.cos_t || a.interleaved ||
                         (a.rotary_dim % 16 == 0 && (half8 & (half8 - 1)) == 0 && (((uintptr_t)a.cos_t | (uintptr_t)a.sin_t) & 31) == 0);
  const bool vec = (a.dim == 32 || a.dim == 64 || a.dim == 128 || a.dim == 256) && a.vdim % 8 == 0 && turn_fits && a.ld % 8 == 0 &&
                   (!a.first || (a.ld_first % 8 == 0 && (uintptr_t)a.first % in_run == 0)) && (uintptr_t)a.proj % in_run == 0 &&
                   (uintptr_t)a.q_out % in_run == 0 && (uintptr_t)kv % kv_run == 0 &&
                   (((uintptr_t)a.bias | (uintptr_t)a.gain_q | (uintptr_t)a.gain_k | (uintptr_t)a.first_bias) & 31) == 0;
  if (!vec) psb_launch(attention_prepare_heads_kernel<T, TKV>, dim3(a.tokens), dim3(PREP_WARPS * 32), 0, stream, a, kv);
  else if (a.dim == 32) launch_heads_vec<T, TKV, 4>(a, kv, stream);
  else if (a.dim == 64) launch_heads_vec<T, TKV, 8>(a, kv, stream);
  else if (a.dim == 128) launch_heads_vec<T, TKV, 16>(a, kv, stream);
  else launch_heads_vec<T, TKV, 32>(a, kv, stream);
}

}  // namespace

// (proj, ld, dtype, positions, token_item, table, table_width, cos, sin, bias, gain_q, gain_k, first, ld_first, first_bias, share,
//  kv, kv_dtype, q_out, T, hq, hkv, dim, vdim, page_size, num_pages, max_positions, rotary_dim, interleaved, eps, split_planes, stream)
PSB_API int psb_attention_prepare_heads(const void* proj, long long ld, int dtype, const void* positions, const void* token_item,
                                        const void* table, int table_width, const void* cos_t, const void* sin_t, const void* bias,
                                        const void* gain_q, const void* gain_k, const void* first, long long ld_first,
                                        const void* first_bias, const void* share, void* kv, int kv_dtype, void* q_out, int T, int hq,
                                        int hkv, int dim, int vdim, int page_size, int num_pages, int max_positions, int rotary_dim,
                                        int interleaved, float eps, int split_planes, cudaStream_t stream) {
  if (T < 0 || hq < 1 || hkv < 1 || dim < 1 || dim > PREP_MAX_D || vdim < 1 || page_size < 1 || table_width < 1 || num_pages < 1)
    PSB_REFUSE("attention_prepare_heads: bad sizes (heads %d/%d, sizes %d/%d, keys of at most %d)", hq, hkv, dim, vdim, PREP_MAX_D);
  if (ld < (long long)(hq + hkv) * dim + (long long)hkv * vdim) PSB_REFUSE("attention_prepare_heads: row stride %lld is shorter than the row", ld);
  if (!(eps > 0.f) || !kv || !table || !gain_q || !gain_k) PSB_REFUSE("attention_prepare_heads: needs a positive eps, gains, the cache entry and the page table");
  if ((cos_t == nullptr) != (sin_t == nullptr)) PSB_REFUSE("attention_prepare_heads: cosines and sines come together");
  if (cos_t && (rotary_dim < 2 || rotary_dim % 2 || rotary_dim > dim || max_positions < 1))
    PSB_REFUSE("attention_prepare_heads: %d rotated elements of %d", rotary_dim, dim);
  if (first && (!share || ld_first < (long long)hkv * vdim)) PSB_REFUSE("attention_prepare_heads: values to mix in need their weight and whole rows");
  if (split_planes && vdim != dim) PSB_REFUSE("attention_prepare_heads: keys and values in planes of their own need vdim == dim, not %d and %d", vdim, dim);
  if (T == 0) return 0;
  PSB_DISPATCH_DTYPE(dtype, T_, {
    HeadsArgs<T_> a{};
    a.proj = (const T_*)proj; a.ld = ld; a.positions = (const int32_t*)positions; a.token_item = (const int32_t*)token_item;
    a.table = (const int32_t*)table; a.table_width = table_width; a.cos_t = (const float*)cos_t; a.sin_t = (const float*)sin_t;
    a.bias = (const float*)bias; a.gain_q = (const float*)gain_q; a.gain_k = (const float*)gain_k; a.first = (const T_*)first;
    a.ld_first = ld_first; a.first_bias = (const float*)first_bias; a.share = (const float*)share; a.q_out = (T_*)q_out; a.tokens = T;
    a.hq = hq; a.hkv = hkv; a.dim = dim; a.vdim = vdim; a.page_size = page_size; a.num_pages = num_pages;
    a.max_positions = max_positions; a.rotary_dim = rotary_dim; a.interleaved = interleaved; a.split_planes = split_planes; a.eps = eps;
    PSB_DISPATCH_DTYPE(kv_dtype, TKV, { launch_heads(a, (TKV*)kv, stream); });
  });
  PSB_LAUNCH_CHECK("attention_prepare_heads");
  return 0;
}

// (proj, ld, dtype, positions, token_item, table, table_width, bias, gain, kv, kv_dtype, q_out, T, hq, hkv, dim, vdim, page_size,
//  num_pages, eps, split_planes, stream); bias (or null) has a number per column of [q | k | v], gain one per column of [q | k]
PSB_API int psb_attention_prepare_normed(const void* proj, long long ld, int dtype, const void* positions, const void* token_item,
                                         const void* table, int table_width, const void* bias, const void* gain, void* kv,
                                         int kv_dtype, void* q_out, int T, int hq, int hkv, int dim, int vdim, int page_size,
                                         int num_pages, float eps, int split_planes, cudaStream_t stream) {
  if (T < 0 || hq < 1 || hkv < 1 || dim < 1 || vdim < 1 || page_size < 1 || table_width < 1 || num_pages < 1)
    PSB_REFUSE("attention_prepare_normed: bad sizes (heads %d/%d, sizes %d/%d)", hq, hkv, dim, vdim);
  if (ld < (long long)(hq + hkv) * dim + (long long)hkv * vdim) PSB_REFUSE("attention_prepare_normed: row stride %lld is shorter than the row", ld);
  if (!(eps > 0.f) || !kv || !table || !gain) PSB_REFUSE("attention_prepare_normed: needs a positive eps, gains, the cache entry and the page table");
  if (split_planes && vdim != dim) PSB_REFUSE("attention_prepare_normed: keys and values in planes of their own need vdim == dim, not %d and %d", vdim, dim);
  if (T == 0) return 0;
  PSB_DISPATCH_DTYPE(dtype, T_, {
    PSB_DISPATCH_DTYPE(kv_dtype, TKV, {
      const bool runs = dim % 8 == 0 && vdim % 8 == 0 && ld % 8 == 0 && (uintptr_t)proj % (8 * sizeof(T_)) == 0 &&
                        (uintptr_t)q_out % (8 * sizeof(T_)) == 0 && (uintptr_t)kv % (8 * sizeof(TKV)) == 0 &&
                        ((uintptr_t)bias | (uintptr_t)gain) % 32 == 0;
      auto launch = [&](auto kernel) {
        psb_launch(kernel, dim3(T), dim3(256), 0, stream, (const T_*)proj, ld, (const int32_t*)positions, (const int32_t*)token_item,
                   (const int32_t*)table, table_width, (const float*)bias, (const float*)gain, (TKV*)kv, (T_*)q_out, hq, hkv, dim,
                   vdim, page_size, num_pages, eps, split_planes);
      };
      if (runs) launch(attention_prepare_normed_kernel<T_, TKV, 8>);
      else launch(attention_prepare_normed_kernel<T_, TKV, 1>);
    });
  });
  PSB_LAUNCH_CHECK("attention_prepare_normed");
  return 0;
}

#define PSB_PREP_ROWS(DD, HH, LL)                                                                                      \
  psb_launch(attention_prepare_rows_kernel<T_, TKV, DD, HH, LL>, dim3((unsigned)blocks), dim3(PREP_WARPS * 32), 0, stream,     \
             (const T_*)proj, ld, (const int32_t*)positions, (const int32_t*)token_item, (const int32_t*)table,        \
             table_width, (const float*)cos_t, (const float*)sin_t, (const float*)head_factor, (TKV*)kv, (T_*)q_out,   \
             hq, hkv, page_size, num_pages, max_positions, rotary_dim, eps, values_are_keys, split_planes, groups)

// (proj, ld, dtype, positions, token_item, table, table_width, cos, sin, head_factor, kv, kv_dtype, q_out, T, hq, hkv, dim, vdim,
//  page_size, num_pages, max_positions, rotary_dim, interleaved, eps, values_are_keys, split_planes, bias, write_kv, stream)
PSB_API int psb_attention_prepare(const void* proj, long long ld, int dtype, const void* positions, const void* token_item, const void* table,
                                  int table_width, const void* cos_t, const void* sin_t, const void* head_factor, void* kv,
                                  int kv_dtype, void* q_out, int T, int hq, int hkv, int dim, int vdim, int page_size,
                                  int num_pages, int max_positions, int rotary_dim, int interleaved, float eps,
                                  int values_are_keys, int split_planes, const void* bias, int write_kv, cudaStream_t stream) {
  if (T < 0 || hq < 1 || hkv < 1 || dim < 1 || dim > PREP_MAX_D || vdim < 1 || page_size < 1 || (write_kv && (table_width < 1 || num_pages < 1)))
    PSB_REFUSE("attention_prepare: bad sizes (heads %d/%d, sizes %d/%d, at most %d)", hq, hkv, dim, vdim, PREP_MAX_D);
  if (write_kv && (!kv || !table)) PSB_REFUSE("attention_prepare: appending keys and values needs the cache entry and the page table");
  if (ld < (long long)hq * dim + (write_kv ? (long long)hkv * dim + (values_are_keys ? 0 : (long long)hkv * vdim) : 0))
    PSB_REFUSE("attention_prepare: row stride %lld is shorter than the row", ld);
  if (values_are_keys && vdim != dim) PSB_REFUSE("attention_prepare: keys that serve as values need vdim == dim, not %d and %d", vdim, dim);
  if ((cos_t == nullptr) != (sin_t == nullptr)) PSB_REFUSE("attention_prepare: cosines and sines come together");
  if (cos_t && (rotary_dim < 2 || rotary_dim % 2 || rotary_dim > dim || max_positions < 1))
    PSB_REFUSE("attention_prepare: %d rotated elements of %d", rotary_dim, dim);
  if (split_planes && vdim != dim) PSB_REFUSE("attention_prepare: keys and values in planes of their own need vdim == dim, not %d and %d", vdim, dim);
  if (T == 0) return 0;
  // heads in registers: sizes that give every lane an even run, a rotation (if any) of neighbours, rows that allow wide loads
  const bool rows_fit = vdim == dim && (dim == 64 || dim == 128 || dim == 256) && (cos_t == nullptr || interleaved) && !bias && write_kv;
  if (rows_fit) {
    // long steps: four heads a warp, their loads in flight together; short ones: a head a warp, as many warps as there are heads
    const int hpw = (long long)T * (hq + hkv) >= 4096 ? 4 : 1;
    // heads of 64 in pairs (16 lanes a head, four elements a lane) when neither the query nor the key heads leave one over
    const int lph = dim == 64 && hq % 2 == 0 && hkv % 2 == 0 ? 16 : 32;
    const int per_block = PREP_WARPS * hpw * (32 / lph);
    const int groups = (hq + hkv + per_block - 1) / per_block;
    const long long blocks = (long long)T * groups;
    bool done = false;
    PSB_DISPATCH_DTYPE(dtype, T_, {
      PSB_DISPATCH_DTYPE(kv_dtype, TKV, {
        const size_t in_run = sizeof(T_) * (size_t)(dim / lph), out_run = sizeof(TKV) * (size_t)(dim / lph);
        if (blocks <= 0x7fffffffLL && (uintptr_t)proj % in_run == 0 && ((size_t)ld * sizeof(T_)) % in_run == 0 &&
            (uintptr_t)q_out % in_run == 0 && (uintptr_t)kv % out_run == 0) {
          if (hpw == 4) {
            if (dim == 64 && lph == 16) PSB_PREP_ROWS(64, 4, 16); else if (dim == 64) PSB_PREP_ROWS(64, 4, 32);
            else if (dim == 128) PSB_PREP_ROWS(128, 4, 32); else PSB_PREP_ROWS(256, 4, 32);
          } else {
            if (dim == 64 && lph == 16) PSB_PREP_ROWS(64, 1, 16); else if (dim == 64) PSB_PREP_ROWS(64, 1, 32);
            else if (dim == 128) PSB_PREP_ROWS(128, 1, 32); else PSB_PREP_ROWS(256, 1, 32);
          }
          done = true;
        }
      });
    });
    if (done) {
      PSB_LAUNCH_CHECK("attention_prepare");
      return 0;
    }
  }
  PSB_DISPATCH_DTYPE(dtype, T_, {
    PSB_DISPATCH_DTYPE(kv_dtype, TKV, {
      psb_launch(attention_prepare_kernel<T_, TKV>, dim3(T), dim3(PREP_WARPS * 32), 0, stream, (const T_*)proj, ld,
                 (const int32_t*)positions, (const int32_t*)token_item, (const int32_t*)table, table_width, (const float*)cos_t,
                 (const float*)sin_t, (const float*)head_factor, (TKV*)kv, (T_*)q_out, hq, hkv, dim, vdim, page_size, num_pages,
                 max_positions, rotary_dim, interleaved, eps, values_are_keys, split_planes, (const float*)bias, write_kv);
    });
  });
  PSB_LAUNCH_CHECK("attention_prepare");
  return 0;
}

// Causal grouped-query attention over the paged cache for designs whose scores carry more than q.k:
//
//   score(i, j) = cap((q_i . k_j) * scale) + bias[h][min(i - j, reach - 1)]  (bias optional; cap(s) = softcap * tanh(s / softcap),
//             optional)
//   visible:  j <= i,  j > i - window (window optional),  floor(j / chunk) == floor(i / chunk) (chunk optional);
//             with ``keep_first`` > 0 (and a window, no chunk) the first keep_first keys of the sequence stay visible
//             to every later query, at their true positions: j <= i and (j > i - window or j < keep_first)
//   weights = exp(score) / (sum over visible j of exp(score) + exp(sink[h]))  (sink optional: a term of the
//             denominator that has no key and no value)
//
//   out = (sum of weights * values) * out_scale * sigmoid(gate)              (gate optional, a number per token, head and value
//             channel; rows of ``out`` and of ``gate`` may be runs of columns of wider ones)
//
// Keys and values may have different sizes (dim, vdim); the cache entry holds one row per token and key/value head,
// [num_pages, 1, hkv, page_size, dim + vdim]: the key, then the value.  ``bias`` is a float32 table
// [heads, reach] by distance (whatever maps distances to learned rows has been applied when the table was built;
// distances of reach - 1 and more share the last column).  Positions are absolute, so the chunk grid is counted
// from the start of the sequence however the prompt was cut.
//
// attention_biased_append_kernel splits a fused projection row [q | k | v] into the query tensor and the cache row.
// attention_biased_kernel: a block per (token, query head) walks the visible keys in runs of 32 aligned to absolute
// positions, its four warps taking the runs in turn, a lane per key for the scores (the key row read 16 bytes at a
// time), online softmax per warp, the four shares and the sink (maximum = sink, sum = 1, no value) joined at the end.
// Scores, weights and sums are float32 and the weights are not rounded before they multiply the values.  Float32 and
// bfloat16 storage.
//
// attention_rows_single_kernel (bfloat16 storage, steps of single tokens): all query heads of a key/value head in one block, the
// scores and the weighted sum on the tensor cores.
//
// attention_biased_tile_kernel (bfloat16 storage): a block takes 16 consecutive tokens of one request and one
// key/value head, with all the query heads that share it; key/value rows are staged in shared memory once for the
// block, a warp takes (token, head) pairs in turn and walks all runs of its pair in order.
#include <cfloat>

#include "common.cuh"

namespace {

constexpr int WARPS = 4;
constexpr int MAX_D = 256;

// The cap on the scores and what is done to a finished row on its way out.
struct RowsTail {
  const void* gate;  // pre-activations of an output gate, rows ldg numbers apart, or null
  long long ldg, ldo;
  float out_scale, softcap;  // softcap 0: none
};

template <typename T>
__device__ __forceinline__ float tail_factor(const RowsTail& tail, size_t t, int column) {
  if (!tail.gate) return tail.out_scale;
  return tail.out_scale / (1.f + expf(-to_float<T>(static_cast<const T*>(tail.gate)[t * tail.ldg + column])));
}

template <typename T, typename TKV>
__global__ void attention_biased_append_kernel(const T* __restrict__ qkv, const int32_t* __restrict__ positions,
                                               const int32_t* __restrict__ token_item, const int32_t* __restrict__ table,
                                               int table_width, TKV* __restrict__ kv, T* __restrict__ q_out, int hq, int hkv,
                                               int dim, int vdim, int page_size, int num_pages) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int qw = hq * dim, kw = hkv * dim, vw = hkv * vdim;
  const T* row = qkv + (size_t)t * (qw + kw + vw);
  for (int c = threadIdx.x; c < qw; c += blockDim.x) q_out[(size_t)t * qw + c] = row[c];
  const int p = positions[t];
  int page = table[(size_t)token_item[t] * table_width + p / page_size];
  if (page < 0 || page >= num_pages) return;  // tables are checked on the host; never write outside the pool
  const int rw = dim + vdim;
  TKV* dst = kv + ((size_t)page * hkv * page_size + (size_t)(p % page_size)) * rw;
  for (int c = threadIdx.x; c < kw + vw; c += blockDim.x) {
    int g, e;
    if (c < kw) { g = c / dim; e = c - g * dim; }
    else { g = (c - kw) / vdim; e = dim + (c - kw) - g * vdim; }
    dst[(size_t)g * page_size * rw + e] = from_float<TKV>(to_float<T>(row[qw + c]));
  }
}

// q . k over ``dim`` elements, 16 bytes of the key row at a time where ``vec`` says the row allows it.
template <typename TKV>
__device__ __forceinline__ float dot_row(const float* __restrict__ q, const TKV* __restrict__ k, int dim, bool vec);
template <>
__device__ __forceinline__ float dot_row<float>(const float* __restrict__ q, const float* __restrict__ k, int dim, bool vec) {
  float dot = 0.f;
  if (vec) {
    for (int d = 0; d < dim; d += 4) {
      const float4 kv = *reinterpret_cast<const float4*>(k + d);
      dot = fmaf(q[d], kv.x, dot); dot = fmaf(q[d + 1], kv.y, dot); dot = fmaf(q[d + 2], kv.z, dot); dot = fmaf(q[d + 3], kv.w, dot);
    }
  } else {
    for (int d = 0; d < dim; ++d) dot = fmaf(q[d], k[d], dot);
  }
  return dot;
}
template <>
__device__ __forceinline__ float dot_row<__nv_bfloat16>(const float* __restrict__ q, const __nv_bfloat16* __restrict__ k, int dim, bool vec) {
  float dot = 0.f;
  if (vec) {
    // four 16-byte pieces of the row are asked for before the first is used (a lane's row is its own: nothing coalesces)
    for (int d0 = 0; d0 < dim; d0 += 32) {
      uint4 raw[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) raw[u] = d0 + 8 * u < dim ? *reinterpret_cast<const uint4*>(k + d0 + 8 * u) : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        if (d0 + 8 * u >= dim) break;
        const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&raw[u]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 kv = __bfloat1622float2(p2[j]);
          dot = fmaf(q[d0 + 8 * u + 2 * j], kv.x, dot);
          dot = fmaf(q[d0 + 8 * u + 2 * j + 1], kv.y, dot);
        }
      }
    }
  } else {
    for (int d = 0; d < dim; ++d) dot = fmaf(q[d], __bfloat162float(k[d]), dot);
  }
  return dot;
}

// A block per (token, query head); its four warps take the runs of 32 keys in turn (run r of the token, counted from
// the aligned start of its visible keys, goes to warp r mod 4) and keep a running maximum, sum and output each; warp 0
// joins the four in warp order.  Which warp gets which run depends on the token's position and the masks only.
template <typename T, typename TKV>
__global__ void __launch_bounds__(WARPS * 32)
attention_biased_kernel(const T* __restrict__ q, const TKV* __restrict__ kv, const int32_t* __restrict__ table,
                        int table_width, const int32_t* __restrict__ positions, const int32_t* __restrict__ token_item,
                        const float* __restrict__ bias, const float* __restrict__ sink, T* __restrict__ out, int T_tokens,
                        int hq, int hkv, int dim, int vdim, int page_size, int window, int chunk, int reach, float scale,
                        const int32_t* __restrict__ item_start, int skip_from, int keep_first, float* __restrict__ partial,
                        int splits, const RowsTail tail) {
  __shared__ __align__(16) float qs[MAX_D];
  __shared__ float part[WARPS][MAX_D + 2];
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x / hq, h = blockIdx.x - t * hq;
  const int g = h / (hq / hkv);
  const int p = positions[t];
  const int item = token_item[t];
  // ``splits`` > 1 (steps of few tokens over many keys): blockIdx.y names this block's share of the runs; it leaves its
  // maximum, sum and unnormalised output in ``partial`` [T * hq, splits, vdim + 2] and the merge kernel joins the shares
  const int split = blockIdx.y;
  if (skip_from > 0 && item_start[item + 1] - item_start[item] >= skip_from) return;  // the tiled kernel's token
  const int32_t* pages = table + (size_t)item * table_width;
  const T* qrow = q + ((size_t)t * hq + h) * dim;
  for (int d = threadIdx.x; d < dim; d += blockDim.x) qs[d] = to_float<T>(qrow[d]);
  __syncthreads();

  int lo = (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0;
  if (chunk > 0) lo = max(lo, (p / chunk) * chunk);
  // kept first keys: when the window still reaches them the visible keys are one stretch from 0; otherwise their runs
  // (counted from key 0) come before the window's runs, and the keys between the two are never touched
  int kept_runs = 0;
  if (keep_first > 0) {
    if (lo <= keep_first) lo = 0;
    else kept_runs = (keep_first + 31) >> 5;
  }
  const int rw = dim + vdim;
  const size_t head_stride = (size_t)page_size * rw;
  const size_t page_elems = (size_t)hkv * head_stride;
  const float* brow = bias ? bias + (size_t)h * reach : nullptr;
  constexpr int PER16 = 16 / (int)sizeof(TKV);
  const bool vec = dim % PER16 == 0 && rw % PER16 == 0 && (((uintptr_t)kv) & 15) == 0;

  float m = -FLT_MAX, l = 0.f;
  float acc[MAX_D / 32];
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) acc[i] = 0.f;

  for (int run = warp + WARPS * split;; run += WARPS * splits) {
    const bool kept = run < kept_runs;
    const int base = kept ? 32 * run : (lo & ~31) + 32 * (run - kept_runs);
    if (base > p) break;
    const int key = base + lane;
    const bool live = kept ? key < keep_first : (key >= lo && key <= p);
    long long off = -1;
    float s = -FLT_MAX;
    if (live) {
      const int page = pages[key / page_size];
      off = (long long)((size_t)page * page_elems + (size_t)g * head_stride + (size_t)(key % page_size) * rw);
      s = dot_row<TKV>(qs, kv + off, dim, vec) * scale;
      if (tail.softcap > 0.f) s = tail.softcap * tanhf(s / tail.softcap);
      if (brow) s += brow[min(p - key, reach - 1)];
    }
    const float m_new = fmaxf(m, warp_max(s));
    const float alpha = expf(m - m_new);
    const float pr = live ? expf(s - m_new) : 0.f;
    l = l * alpha + warp_sum(pr);
    m = m_new;
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) acc[i] *= alpha;
    const int n_live = kept ? min(32, keep_first - base) : min(32, p - base + 1);
    // eight keys at a time: their value rows are asked for together, then added in key order
    for (int j0 = 0; j0 < n_live; j0 += 8) {
      float pj[8];
      long long oj[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        pj[k] = __shfl_sync(0xffffffffu, pr, (j0 + k) & 31);
        oj[k] = __shfl_sync(0xffffffffu, off, (j0 + k) & 31);
      }
#pragma unroll
      for (int i = 0; i < MAX_D / 32; ++i) {
        const int d = lane + 32 * i;
        if (d < vdim) {
          float v[8];
#pragma unroll
          for (int k = 0; k < 8; ++k) v[k] = oj[k] >= 0 ? to_float<TKV>(kv[oj[k] + dim + d]) : 0.f;
#pragma unroll
          for (int k = 0; k < 8; ++k) acc[i] = fmaf(pj[k], v[k], acc[i]);
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) {
    const int d = lane + 32 * i;
    if (d < vdim) part[warp][d] = acc[i];
  }
  if (lane == 0) { part[warp][MAX_D] = m; part[warp][MAX_D + 1] = l; }
  __syncthreads();
  if (warp != 0) return;
  // join: the sink first (maximum = sink, sum = 1, no value; with split keys it joins in the merge kernel), then the warps in order
  const bool sink_here = sink && splits == 1;
  float M = sink_here ? sink[h] : -FLT_MAX, L = sink_here ? 1.f : 0.f;
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) acc[i] = 0.f;
  for (int w = 0; w < WARPS; ++w) {
    const float mw = part[w][MAX_D], lw = part[w][MAX_D + 1];
    if (lw == 0.f) continue;  // a warp without keys
    const float m_new = fmaxf(M, mw);
    const float a = expf(M - m_new), b2 = expf(mw - m_new);
    L = L * a + lw * b2;
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) {
      const int d = lane + 32 * i;
      if (d < vdim) acc[i] = acc[i] * a + part[w][d] * b2;
    }
    M = m_new;
  }
  if (splits > 1) {
    float* mine = partial + (((size_t)t * hq + h) * splits + split) * (vdim + 2);
    if (lane == 0) { mine[0] = M; mine[1] = L; }
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) {
      const int d = lane + 32 * i;
      if (d < vdim) mine[2 + d] = acc[i];
    }
    return;
  }
  const float inv = 1.f / L;
  T* orow = out + (size_t)t * tail.ldo + (size_t)h * vdim;
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) {
    const int d = lane + 32 * i;
    if (d < vdim) orow[d] = from_float<T>(acc[i] * inv * tail_factor<T>(tail, t, h * vdim + d));
  }
}

// Joins the shares of the blocks that split a (token, head)'s runs among them, in split order, the sink first.
constexpr int MAX_KEY_SPLITS = 16;

template <typename T>
__global__ void __launch_bounds__(32)
attention_biased_merge_kernel(const float* __restrict__ partial, const float* __restrict__ sink, T* __restrict__ out, int hq,
                              int vdim, int splits, const RowsTail tail) {
  pdl_trigger();
  pdl_wait();
  const size_t unit = blockIdx.x;  // token * hq + head
  const int lane = threadIdx.x, h = (int)(unit % hq);
  const float* mine = partial + unit * splits * (vdim + 2);
  // every share's maximum and sum are asked for at once, then every share's output: nothing here waits for a share before
  // it asks for the next
  float ms[MAX_KEY_SPLITS], ls[MAX_KEY_SPLITS];
#pragma unroll
  for (int s = 0; s < MAX_KEY_SPLITS; ++s) {
    ms[s] = s < splits ? mine[(size_t)s * (vdim + 2)] : -FLT_MAX;
    ls[s] = s < splits ? mine[(size_t)s * (vdim + 2) + 1] : 0.f;
  }
  float M = sink ? sink[h] : -FLT_MAX;
#pragma unroll
  for (int s = 0; s < MAX_KEY_SPLITS; ++s)
    if (ls[s] > 0.f) M = fmaxf(M, ms[s]);  // (a share without keys has a sum of zero)
  float L = sink ? expf(sink[h] - M) : 0.f;
  float acc[MAX_D / 32];
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) acc[i] = 0.f;
#pragma unroll
  for (int s = 0; s < MAX_KEY_SPLITS; ++s) {
    if (s >= splits) break;
    const float f = ls[s] > 0.f ? expf(ms[s] - M) : 0.f;
    L += ls[s] * f;
    const float* share = mine + (size_t)s * (vdim + 2) + 2;
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) {
      const int d = lane + 32 * i;
      if (d < vdim) acc[i] = fmaf(share[d], f, acc[i]);
    }
  }
  const float inv = 1.f / L;
  const size_t t = unit / hq;
  T* orow = out + t * tail.ldo + (size_t)h * vdim;
#pragma unroll
  for (int i = 0; i < MAX_D / 32; ++i) {
    const int d = lane + 32 * i;
    if (d < vdim) orow[d] = from_float<T>(acc[i] * inv * tail_factor<T>(tail, t, h * vdim + d));
  }
}

// Prompt portions in bfloat16: a block = up to TILE_T consecutive tokens of one item x one key/value head.  The keys a
// tile can see lie in [lo of its first token, position of its last]; they are brought into shared memory 32 at a time
// (the same absolute runs of 32 the kernel above walks), transposed so that a lane's key is a column, and every
// (token, query head) pair of the tile, one warp each in turn, works on the staged run.
constexpr int TILE_T = 16;
constexpr int TILE_WARPS = 8;

template <int DP, int VP>  // key and value sizes rounded up to 32, 64, 128 or 256
__global__ void __launch_bounds__(TILE_WARPS * 32)
attention_biased_tile_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ kv,
                             const int32_t* __restrict__ table, int table_width, const int32_t* __restrict__ positions,
                             const int32_t* __restrict__ item_start, int items, int min_tokens, const float* __restrict__ bias,
                             const float* __restrict__ sink, __nv_bfloat16* __restrict__ out, int hq, int hkv, int dim, int vdim,
                             int page_size, int window, int chunk, int reach, float scale, int keep_first, const RowsTail tail) {
  extern __shared__ float smem[];
  pdl_trigger();
  pdl_wait();
  // tiles are numbered through the portions of at least ``min_tokens`` tokens, in order
  int item = -1, t0 = 0;
  for (int i = 0, left = blockIdx.x; i < items; ++i) {
    const int a = item_start[i], n = item_start[i + 1] - a;
    if (n < min_tokens) continue;
    const int tiles = (n + TILE_T - 1) / TILE_T;
    if (left < tiles) { item = i; t0 = a + left * TILE_T; break; }
    left -= tiles;
  }
  if (item < 0) return;
  const int g = blockIdx.y, share = hq / hkv;
  const int nt = min(TILE_T, item_start[item + 1] - t0);
  const int pairs = nt * share;  // (token, head of the group) units of this block
  float* ks = smem;                               // [DP][33] one run of keys, transposed
  float* vs = ks + DP * 33;                       // [32][VP]
  float* qs = vs + 32 * VP;                       // [TILE_T * share][DP]
  float* st = qs + (size_t)TILE_T * share * DP;   // per unit: m, l
  float* accs = st + 2 * TILE_T * share;          // [TILE_T * share][VP]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rw = dim + vdim;
  const size_t head_stride = (size_t)page_size * rw;
  const size_t page_elems = (size_t)hkv * head_stride;
  const int32_t* pages = table + (size_t)item * table_width;
  const int p_first = positions[t0], p_last = p_first + nt - 1;
  for (int i = threadIdx.x; i < pairs * DP; i += blockDim.x) {
    const int u = i / DP, d = i - u * DP;
    const int tt = u / share, hh = g * share + (u - tt * share);
    qs[i] = d < dim ? __bfloat162float(q[((size_t)(t0 + tt) * hq + hh) * dim + d]) : 0.f;
  }
  for (int i = threadIdx.x; i < pairs * VP; i += blockDim.x) accs[i] = 0.f;
  for (int u = threadIdx.x; u < pairs; u += blockDim.x) {
    const int hh = g * share + u % share;
    st[2 * u] = sink ? sink[hh] : -FLT_MAX;
    st[2 * u + 1] = sink ? 1.f : 0.f;
  }
  int lo_tile = (window > 0 && p_first - window + 1 > 0) ? p_first - window + 1 : 0;
  if (chunk > 0) lo_tile = max(lo_tile, (p_first / chunk) * chunk);
  // kept first keys: one stretch from 0 while the tile's first token still reaches them; else their runs come first
  // (then every token of the tile has a gap between the kept keys and its window)
  int kept_runs = 0;
  if (keep_first > 0) {
    if (lo_tile <= keep_first) lo_tile = 0;
    else kept_runs = (keep_first + 31) >> 5;
  }
  for (int run = 0;; ++run) {
    const bool kept = run < kept_runs;
    const int base = kept ? 32 * run : (lo_tile & ~31) + 32 * (run - kept_runs);
    if (base > p_last) break;
    __syncthreads();
    // stage the run: keys transposed, values as rows; a key beyond the tile's last position is left as zeros
    for (int i = threadIdx.x; i < 32 * (DP + VP) / 2; i += blockDim.x) {
      const int j = i / ((DP + VP) / 2), e = 2 * (i - j * ((DP + VP) / 2));
      const int key = base + j;
      float a = 0.f, b = 0.f;
      const bool is_key = e < DP;
      const int col = is_key ? e : e - DP;
      const int width = is_key ? dim : vdim;
      if ((kept ? key < keep_first : (key >= lo_tile && key <= p_last)) && col < width) {
        const int page = pages[key / page_size];
        const __nv_bfloat16* src = kv + (size_t)page * page_elems + (size_t)g * head_stride + (size_t)(key % page_size) * rw +
                                   (is_key ? 0 : dim) + col;
        a = __bfloat162float(src[0]);
        if (col + 1 < width) b = __bfloat162float(src[1]);
      }
      if (is_key) { ks[col * 33 + j] = a; ks[(col + 1) * 33 + j] = b; }
      else { vs[j * VP + col] = a; vs[j * VP + col + 1] = b; }
    }
    __syncthreads();
    for (int u = warp; u < pairs; u += TILE_WARPS) {
      const int tt = u / share, hh = g * share + (u - tt * share);
      const int p = p_first + tt;
      if (base > p) continue;
      int lo = (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0;
      if (chunk > 0) lo = max(lo, (p / chunk) * chunk);
      if (keep_first > 0 && lo <= keep_first) lo = 0;
      // (a tile whose first token still reaches the kept keys has no kept runs, but a later token's window may
      // already start beyond them: such a token sees the kept keys inside the ordinary runs)
      const bool inline_kept = kept_runs == 0 && keep_first > 0;  // the kept keys lie inside the ordinary runs
      if (!kept && base + 31 < lo && !(inline_kept && base < keep_first)) continue;
      const int key = base + lane;
      const bool live = kept ? key < keep_first : (key <= p && (key >= lo || (inline_kept && key < keep_first)));
      float s = -FLT_MAX;
      if (live) {
        const float* qq = qs + (size_t)u * DP;
        float dot = 0.f;
        for (int d = 0; d < dim; ++d) dot = fmaf(qq[d], ks[d * 33 + lane], dot);
        s = dot * scale;
        if (tail.softcap > 0.f) s = tail.softcap * tanhf(s / tail.softcap);
        if (bias) s += bias[(size_t)hh * reach + min(p - key, reach - 1)];
      }
      float m = st[2 * u], l = st[2 * u + 1];
      const float m_new = fmaxf(m, warp_max(s));
      const float alpha = expf(m - m_new);
      const float pr = live ? expf(s - m_new) : 0.f;
      l = l * alpha + warp_sum(pr);
      __syncwarp();
      if (lane == 0) { st[2 * u] = m_new; st[2 * u + 1] = l; }
      float* acc = accs + (size_t)u * VP;
      float a[VP / 32];
#pragma unroll
      for (int i = 0; i < VP / 32; ++i) a[i] = acc[lane + 32 * i] * alpha;
      const int n_live = kept ? min(32, keep_first - base) : min(32, p - base + 1);
      const int j0 = (kept || (inline_kept && base < keep_first)) ? 0 : max(0, lo - base);
      for (int j = j0; j < n_live; ++j) {
        const float pj = __shfl_sync(0xffffffffu, pr, j);
#pragma unroll
        for (int i = 0; i < VP / 32; ++i) a[i] = fmaf(pj, vs[j * VP + lane + 32 * i], a[i]);
      }
#pragma unroll
      for (int i = 0; i < VP / 32; ++i) acc[lane + 32 * i] = a[i];
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < pairs * VP; i += blockDim.x) {
    const int u = i / VP, d = i - u * VP;
    if (d >= vdim) continue;
    const int tt = u / share, hh = g * share + (u - tt * share);
    out[(size_t)(t0 + tt) * tail.ldo + (size_t)hh * vdim + d] =
        __float2bfloat16_rn(accs[i] / st[2 * u + 1] * tail_factor<__nv_bfloat16>(tail, t0 + tt, hh * vdim + d));
  }
}

__device__ __forceinline__ void mma_16816(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat16 ha = __float2bfloat16_rn(a), hb = __float2bfloat16_rn(b);
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - __bfloat162float(ha), b - __bfloat162float(hb));
}

__device__ __forceinline__ void rows_ldmatrix4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void rows_ldmatrix4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void rows_copy16(uint32_t dst, const void* src, bool there) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(there ? 16 : 0) : "memory");
}

// elements between the rows of a ring: an odd number of 16-byte pieces, so that ldmatrix meets every bank once
__host__ __device__ __forceinline__ int rows_pitch(int row) { return (row / 8) % 2 ? row : row + 8; }
// cap * tanh(x / cap) with x = s * scale, as cap - 2 cap / (exp(2 x / cap) + 1): an error of a few units in the last place of the
// cap, and far out it reaches +-cap.  ``rate`` = 2 log2(e) scale / cap.
__device__ __forceinline__ float quick_cap(float s, float rate, float cap) { return fmaf(-2.f * cap, __fdividef(1.f, exp2f(s * rate) + 1.f), cap); }

// Prompt portions in bfloat16 on the tensor cores (mma.sync m16n8k16, float32 sums): a block of eight warps takes 128 (token, query
// head) rows of one request, a warp 16 tokens of one head: 128 consecutive tokens of one head, or 64 of two heads that read the
// same keys and values.  Keys come in blocks of 64 aligned to absolute positions, whole cache rows (key, then value) brought in
// with cp.async one block ahead of the arithmetic (zeros for keys outside the tile's reach, so nothing of a page that was never
// written is read) and worked on 32 at a time; the queries stay in shared memory, so that two blocks fit an SM.  S = Q K^T stays in the accumulator registers, where scale, cap, bias, masks and the online softmax (powers of
// two, started from the sink) are applied in float32; the weights enter the second product as the sum of two bfloat16 numbers
// (p = hi + lo, two instructions), so they keep 16 bits.  Late tiles (of a sequence or of its chunks), which see
// the most keys, are started first.
constexpr int MMA_WARPS = 8, MMA_KEYS = 64, MMA_PART = 32;
constexpr int MMA_BIAS = 1024;  // distances whose bias a block keeps in shared memory, per head

inline size_t mma_smem(int dim, int vdim, bool bias, int heads) {
  return (size_t)2 * MMA_KEYS * rows_pitch(dim + vdim) * 2 + 32 + (size_t)16 * MMA_WARPS * rows_pitch((dim + 15) / 16 * 16) * 2 + (bias ? (size_t)heads * MMA_BIAS * 4 : 0);
}

template <int D, int V>  // key and value sizes rounded up to 64 or 128
__global__ void __launch_bounds__(MMA_WARPS * 32, 2)
attention_biased_mma_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ kv,
                            const int32_t* __restrict__ table, int table_width, const int32_t* __restrict__ positions,
                            const int32_t* __restrict__ item_start, int items, int min_tokens, const float* __restrict__ bias,
                            const float* __restrict__ sink, __nv_bfloat16* __restrict__ out, int hq, int hkv, int dim, int vdim,
                            int page_size, int window, int chunk, int reach, float scale, int keep_first, int heads_here, const RowsTail tail) {
  extern __shared__ __align__(16) unsigned char mma_raw[];
  pdl_wait();
  const int tile_tokens = 16 * MMA_WARPS / heads_here;
  int item = -1, t0 = 0, tiles = 0;
  for (int i = 0; i < items; ++i) {
    const int n = item_start[i + 1] - item_start[i];
    if (n >= min_tokens) tiles += (n + tile_tokens - 1) / tile_tokens;
  }
  int at = tiles - 1 - (int)blockIdx.y;
  if (chunk >= 2 * tile_tokens && items == 1) {  // (the launch has blocks for this): the late tiles of every chunk, then the ones before them
    const int per = chunk / tile_tokens, chunks = (tiles + per - 1) / per, round = (int)blockIdx.y / chunks;
    at = ((int)blockIdx.y - round * chunks) * per + per - 1 - round;
    if (round >= per || at >= tiles) return;
  }
  for (int i = 0, left = at; i < items && left >= 0; ++i) {
    const int a = item_start[i], n = item_start[i + 1] - a;
    if (n < min_tokens) continue;
    const int mine = (n + tile_tokens - 1) / tile_tokens;
    if (left < mine) { item = i; t0 = a + left * tile_tokens; break; }
    left -= mine;
  }
  if (item < 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int warps_a_head = MMA_WARPS / heads_here;
  const int h0 = blockIdx.x * heads_here, which = warp / warps_a_head, h = h0 + which, g = h / (hq / hkv);
  const int row0 = (warp - which * warps_a_head) * 16;  // this warp's first token of the tile
  const int nt = min(tile_tokens, item_start[item + 1] - t0);
  const int rw = dim + vdim, pitch = rows_pitch(rw), pieces = rw / 8;
  const size_t head_stride = (size_t)page_size * rw, page_elems = (size_t)hkv * head_stride;
  const int32_t* pages = table + (size_t)item * table_width;
  const int p_first = positions[t0], p_last = p_first + nt - 1;
  const uint32_t ring = (uint32_t)__cvta_generic_to_shared(mma_raw);
  const int q_width = (dim + 15) / 16 * 16, q_pitch = rows_pitch(q_width);
  unsigned char* q_raw = mma_raw + (size_t)2 * MMA_KEYS * pitch * 2 + 32;  // the warps' queries, 16 rows each
  float* near_bias = reinterpret_cast<float*>(q_raw + (size_t)16 * MMA_WARPS * q_pitch * 2);  // the heads' bias for the nearest distances

  int lo_tile = (window > 0 && p_first - window + 1 > 0) ? p_first - window + 1 : 0;
  if (chunk > 0) lo_tile = max(lo_tile, (p_first / chunk) * chunk);
  // kept first keys: one stretch from 0 while the tile's first token still reaches them; else their blocks come first
  int kept_blocks = 0;
  if (keep_first > 0) {
    if (lo_tile <= keep_first) lo_tile = 0;
    else kept_blocks = (keep_first + MMA_KEYS - 1) / MMA_KEYS;
  }
  const int blocks = kept_blocks + p_last / MMA_KEYS - lo_tile / MMA_KEYS + 1;
  auto base_of = [&](int blk) { return MMA_KEYS * (blk < kept_blocks ? blk : lo_tile / MMA_KEYS + blk - kept_blocks); };
  auto fetch = [&](int blk) {
    if (blk < blocks) {
      const int base = base_of(blk) + warp * (MMA_KEYS / MMA_WARPS);
      long long off = -1;  // lane r: where this warp's row r of the block lies
      if (lane < MMA_KEYS / MMA_WARPS) {
        const int key = base + lane;
        if (blk < kept_blocks ? key < keep_first : (key >= lo_tile && key <= p_last))
          off = (long long)((size_t)pages[key / page_size] * page_elems + (size_t)g * head_stride + (size_t)(key % page_size) * rw);
      }
      const uint32_t dst = ring + (uint32_t)(((blk & 1) * MMA_KEYS + warp * (MMA_KEYS / MMA_WARPS)) * pitch * 2);
#pragma unroll
      for (int r = 0; r < MMA_KEYS / MMA_WARPS; ++r) {
        const long long at = __shfl_sync(0xffffffffu, off, r);
        for (int c = lane; c < pieces; c += 32) rows_copy16(dst + (uint32_t)(r * pitch + c * 8) * 2, kv + (at < 0 ? 0 : at) + c * 8, at >= 0);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);

  // a warp brings in its own queries and is the only one to read them (rows beyond the portion and columns beyond dim are zeros)
  for (int i = lane; i < 16 * (q_width / 8); i += 32) {
    const int r = i / (q_width / 8), c = (i - r * (q_width / 8)) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row0 + r < nt && c < dim) v = *reinterpret_cast<const uint4*>(q + ((size_t)(t0 + row0 + r) * hq + h) * dim + c);
    *reinterpret_cast<uint4*>(q_raw + (size_t)((warp * 16 + r) * q_pitch + c) * 2) = v;
  }
  __syncwarp();
  // this thread's two rows: positions, lowest visible keys, running maximum and its share of the running sum
  int pos[2], low[2];
  float m[2], l[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    pos[r] = p_first + row0 + gid + 8 * r;
    low[r] = (window > 0 && pos[r] - window + 1 > 0) ? pos[r] - window + 1 : 0;
    if (chunk > 0) low[r] = max(low[r], (pos[r] / chunk) * chunk);
    if (keep_first > 0 && low[r] <= keep_first) low[r] = 0;
    m[r] = sink ? sink[h] * PSB_LOG2E : -FLT_MAX;
    l[r] = (sink && tig == 0) ? 1.f : 0.f;
  }
  // what the warp's rows see as a whole: every key of [all_from, all_to], none below none_below (the lowest is the first row's)
  const int w_first = p_first + row0, w_last = w_first + 15;
  const int none_below = __shfl_sync(0xffffffffu, low[0], 0), all_from = __shfl_sync(0xffffffffu, low[1], 31), all_to = w_first;
  float o[V / 8][4];
#pragma unroll
  for (int i = 0; i < V / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  if (bias)
    for (int i = threadIdx.x; i < heads_here * MMA_BIAS; i += MMA_WARPS * 32) {
      const int d = i % MMA_BIAS;
      near_bias[i] = d < reach ? bias[(size_t)(h0 + i / MMA_BIAS) * reach + d] * PSB_LOG2E : 0.f;  // visible after the loop's first barrier
    }
  const float* brow = bias ? bias + (size_t)h * reach : nullptr;
  const float factor = scale * PSB_LOG2E, cap = tail.softcap * PSB_LOG2E, rate = tail.softcap > 0.f ? 2.f * PSB_LOG2E * scale / tail.softcap : 0.f;
  const int lrow = lane & 7, lmat = lane >> 3;
  const uint32_t q_at = (uint32_t)__cvta_generic_to_shared(q_raw) + (uint32_t)((warp * 16 + (lmat & 1) * 8 + lrow) * q_pitch + (lmat >> 1) * 8) * 2;

  for (int blk = 0; blk < blocks; ++blk) {
    const bool kept = blk < kept_blocks;
    const int base = base_of(blk);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this block has landed for everybody, and everybody is done with the other buffer
    fetch(blk + 1);
    // no rows, or all of them before the block or (without kept keys) beyond what they see (uniform in the warp)
    if (row0 >= nt || base > w_last || (keep_first == 0 && base + MMA_KEYS - 1 < none_below)) continue;
#pragma unroll 1
    for (int part = 0; part < MMA_KEYS; part += MMA_PART) {
      const int key0 = base + part;
      if (key0 > w_last || (keep_first == 0 && key0 + MMA_PART - 1 < none_below)) continue;
      const uint32_t src = ring + (uint32_t)(((blk & 1) * MMA_KEYS + part) * pitch * 2);
      float sc[MMA_PART / 8][4];
#pragma unroll
      for (int n = 0; n < MMA_PART / 8; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < D / 16; ++kk) {
        if (kk * 16 >= dim) break;  // (keys in an odd number of eights: the last step meets value channels with zeros of q)
        uint32_t a[4];
        rows_ldmatrix4(a, q_at + (uint32_t)(kk * 32));
#pragma unroll
        for (int n = 0; n < MMA_PART / 8; n += 2) {
          uint32_t b[4];
          rows_ldmatrix4(b, src + (uint32_t)((n * 8 + (lmat >> 1) * 8 + lrow) * pitch + kk * 16 + (lmat & 1) * 8) * 2);
          mma_16816(sc[n], a[0], a[1], a[2], a[3], b[0], b[1]);
          mma_16816(sc[n + 1], a[0], a[1], a[2], a[3], b[2], b[3]);
        }
      }
      if (tail.softcap > 0.f) {
#pragma unroll
        for (int n = 0; n < MMA_PART / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) sc[n][e] = quick_cap(sc[n][e], rate, cap);
      } else {
#pragma unroll
        for (int n = 0; n < MMA_PART / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) sc[n][e] *= factor;
      }
      if (brow) {
#pragma unroll
        for (int n = 0; n < MMA_PART / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int far = max(0, min(pos[e >> 1] - (key0 + n * 8 + 2 * tig + (e & 1)), reach - 1));
            sc[n][e] += far < MMA_BIAS ? near_bias[which * MMA_BIAS + far] : brow[far] * PSB_LOG2E;
          }
      }
      if (kept || key0 < all_from || key0 + MMA_PART - 1 > all_to) {
        // (without kept blocks of their own the kept keys lie inside the ordinary blocks: a later row of the tile may see them
        // although its window starts beyond them; a kept block lies before every row of a tile that has any)
#pragma unroll
        for (int n = 0; n < MMA_PART / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int r = e >> 1, key = key0 + n * 8 + 2 * tig + (e & 1);
            if (!(kept ? key < keep_first : (key <= pos[r] && (key >= low[r] || (kept_blocks == 0 && key < keep_first))))) sc[n][e] = -INFINITY;
          }
      }
      float top[2] = {m[0], m[1]};
#pragma unroll
      for (int n = 0; n < MMA_PART / 8; ++n) {
        top[0] = fmaxf(top[0], fmaxf(sc[n][0], sc[n][1]));
        top[1] = fmaxf(top[1], fmaxf(sc[n][2], sc[n][3]));
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 1));
        top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 2));
      }
      if (__any_sync(0xffffffffu, top[0] > m[0] || top[1] > m[1])) {  // a row's maximum has grown (multiplying by one else)
        const float alpha[2] = {exp2f(m[0] - top[0]), exp2f(m[1] - top[1])};
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          m[r] = top[r];
          l[r] *= alpha[r];
        }
#pragma unroll
        for (int i = 0; i < V / 8; ++i) {
          o[i][0] *= alpha[0]; o[i][1] *= alpha[0];
          o[i][2] *= alpha[1]; o[i][3] *= alpha[1];
        }
      }
#pragma unroll
      for (int kk = 0; kk < MMA_PART / 16; ++kk) {
#pragma unroll
        for (int n = 2 * kk; n < 2 * kk + 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            sc[n][e] = exp2f(sc[n][e] - m[e >> 1]);  // a masked score is -inf: weight 0
            l[e >> 1] += sc[n][e];
          }
        uint32_t hi[4], lo[4];
        split_bf16(sc[2 * kk][0], sc[2 * kk][1], hi[0], lo[0]);
        split_bf16(sc[2 * kk][2], sc[2 * kk][3], hi[1], lo[1]);
        split_bf16(sc[2 * kk + 1][0], sc[2 * kk + 1][1], hi[2], lo[2]);
        split_bf16(sc[2 * kk + 1][2], sc[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int nv = 0; nv < V / 8; nv += 2) {
          if (nv * 8 >= vdim) break;
          uint32_t b[4];  // (values in an odd number of eights: the last columns read 16 bytes beyond the row, and nobody stores them)
          rows_ldmatrix4_trans(b, src + (uint32_t)((kk * 16 + (lmat & 1) * 8 + lrow) * pitch + dim + nv * 8 + (lmat >> 1) * 8) * 2);
          mma_16816(o[nv], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
          mma_16816(o[nv + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
          mma_16816(o[nv], lo[0], lo[1], lo[2], lo[3], b[0], b[1]);
          mma_16816(o[nv + 1], lo[0], lo[1], lo[2], lo[3], b[2], b[3]);
        }
      }
    }
  }
  pdl_trigger();  // late: blocks of the next kernel waiting beside this one's few warps would only be in their way
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = row0 + gid + 8 * r;
    if (row >= nt) continue;
    const float inv = 1.f / l[r];
    __nv_bfloat16* orow = out + (size_t)(t0 + row) * tail.ldo + (size_t)h * vdim;
#pragma unroll
    for (int nv = 0; nv < V / 8; ++nv) {
      const int c = nv * 8 + 2 * tig;
      if (c < vdim)
        *reinterpret_cast<uint32_t*>(orow + c) = pack_bf16(o[nv][2 * r] * (inv * tail_factor<__nv_bfloat16>(tail, t0 + row, h * vdim + c)),
                                                           o[nv][2 * r + 1] * (inv * tail_factor<__nv_bfloat16>(tail, t0 + row, h * vdim + c + 1)));
    }
  }
}

// Steps of single tokens in bfloat16 on the tensor cores: a block of four warps takes a token, a key/value head with up to 16 of
// the query heads that read it, and a share of the keys.  Keys come in runs of 16 aligned to absolute positions; run r goes to
// share (r / 4) mod splits, warp r mod 4, and every warp brings its own runs in with cp.async through a ring of its own, whole
// cache rows (key, then value) at a time; a row outside the masks is zeros.  S = Q K^T (mma.sync m16n8k16: heads in rows, keys in
// columns) stays in registers, where scale, cap, bias, masks and the online softmax are applied in float32; the weights enter the
// second product as the sum of two bfloat16 numbers.  The warps are joined in warp order; with several shares the merge kernel
// above joins them.
constexpr int ROWS_WARPS = 4, ROWS_RUN = 16, ROWS_HEADS = 16, ROWS_STAGES = 3;

inline size_t rows_smem(int dim, int vdim) {
  const size_t ring = (size_t)ROWS_WARPS * ROWS_STAGES * ROWS_RUN * rows_pitch(dim + vdim) * 2 + 32;
  const size_t join = (size_t)ROWS_WARPS * ROWS_HEADS * (vdim + 2) * 4;
  return ring > join ? ring : join;
}

template <int D, int V>  // key and value sizes rounded up to 64 or 128
__global__ void __launch_bounds__(ROWS_WARPS * 32)
attention_rows_single_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ kv, const int32_t* __restrict__ table,
                             int table_width, const int32_t* __restrict__ positions, const int32_t* __restrict__ token_item,
                             const float* __restrict__ bias, const float* __restrict__ sink, __nv_bfloat16* __restrict__ out, int hq, int hkv,
                             int dim, int vdim, int page_size, int window, int chunk, int reach, float scale, int keep_first,
                             float* __restrict__ partial, int splits, const RowsTail tail) {
  extern __shared__ __align__(16) unsigned char rows_raw[];
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int share = hq / hkv, groups = (share + ROWS_HEADS - 1) / ROWS_HEADS;
  const int t = blockIdx.x / (hkv * groups), rest = blockIdx.x - t * hkv * groups;
  const int g = rest / groups, h0 = g * share + (rest - g * groups) * ROWS_HEADS;
  const int heads = min(ROWS_HEADS, (g + 1) * share - h0);
  // inputs of the step: they may be read before the preceding kernel has finished
  const int p = positions[t];
  const int32_t* pages = table + (size_t)token_item[t] * table_width;
  int lo = (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0;
  if (chunk > 0) lo = max(lo, (p / chunk) * chunk);
  int kept_runs = 0;  // kept first keys: one stretch from 0 while the window reaches them, else runs of their own in front
  if (keep_first > 0) {
    if (lo <= keep_first) lo = 0;
    else kept_runs = (keep_first + ROWS_RUN - 1) / ROWS_RUN;
  }
  const int first_run = lo / ROWS_RUN, runs = kept_runs + p / ROWS_RUN - first_run + 1;
  const int rw = dim + vdim, pitch = rows_pitch(rw), pieces = rw / 8;
  const size_t head_stride = (size_t)page_size * rw, page_elems = (size_t)hkv * head_stride;
  const uint32_t ring = (uint32_t)__cvta_generic_to_shared(rows_raw) + (uint32_t)(warp * ROWS_STAGES * ROWS_RUN * pitch * 2);
  const int step = ROWS_WARPS * splits, mine = blockIdx.y * ROWS_WARPS + warp;
  auto base_of = [&](int run) { return ROWS_RUN * (run < kept_runs ? run : first_run + run - kept_runs); };
  pdl_wait();  // queries and this step's cache rows are the preceding kernels' output

  auto fetch = [&](int run, int stage) {
    if (run < runs) {
      const int base = base_of(run);
      long long off = -1;  // lane r: where row r of the run lies
      if (lane < ROWS_RUN) {
        const int key = base + lane;
        if (run < kept_runs ? key < keep_first : (key >= lo && key <= p))
          off = (long long)((size_t)pages[key / page_size] * page_elems + (size_t)g * head_stride + (size_t)(key % page_size) * rw);
      }
      const uint32_t dst = ring + (uint32_t)(stage * ROWS_RUN * pitch * 2);
#pragma unroll 4
      for (int r = 0; r < ROWS_RUN; ++r) {
        const long long at = __shfl_sync(0xffffffffu, off, r);
        for (int c = lane; c < pieces; c += 32) rows_copy16(dst + (uint32_t)(r * pitch + c * 8) * 2, kv + (at < 0 ? 0 : at) + c * 8, at >= 0);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int s = 0; s < ROWS_STAGES - 1; ++s) fetch(mine + s * step, s);

  // the heads' queries as operand fragments (rows beyond the heads are zeros)
  uint32_t qf[D / 16][4];
#pragma unroll
  for (int kk = 0; kk < D / 16; ++kk)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int row = gid + 8 * (e & 1), c = kk * 16 + 2 * tig + 8 * (e >> 1);
      qf[kk][e] = row < heads && c < dim ? *reinterpret_cast<const uint32_t*>(q + ((size_t)t * hq + h0 + row) * dim + c) : 0u;
    }
  float m[2] = {-FLT_MAX, -FLT_MAX}, l[2] = {0.f, 0.f};
  float o[V / 8][4];
#pragma unroll
  for (int i = 0; i < V / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  const int lrow = lane & 7, lmat = lane >> 3;
  const float rate = tail.softcap > 0.f ? 2.f * PSB_LOG2E * scale / tail.softcap : 0.f;
  int stage = 0;
  for (int run = mine; run < runs; run += step) {
    asm volatile("cp.async.wait_group %0;" ::"n"(ROWS_STAGES - 2) : "memory");
    __syncwarp();  // every lane's copies of this run have landed, and every lane is done with the run before
    fetch(run + (ROWS_STAGES - 1) * step, stage == 0 ? ROWS_STAGES - 1 : stage - 1);
    const uint32_t src = ring + (uint32_t)(stage * ROWS_RUN * pitch * 2);
    stage = stage + 1 == ROWS_STAGES ? 0 : stage + 1;
    float sc[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      if (kk * 16 >= dim) break;
      uint32_t b[4];
      rows_ldmatrix4(b, src + (uint32_t)(((lmat >> 1) * 8 + lrow) * pitch + kk * 16 + (lmat & 1) * 8) * 2);
      mma_16816(sc[0], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], b[0], b[1]);
      mma_16816(sc[1], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], b[2], b[3]);
    }
    const bool kept = run < kept_runs;
    const int base = base_of(run);
    float top[2] = {-FLT_MAX, -FLT_MAX};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = e >> 1, key = base + n * 8 + 2 * tig + (e & 1);
        if (r == 1 && heads <= 8) break;  // no heads in the upper rows (the same for the whole block)
        float v = tail.softcap > 0.f ? quick_cap(sc[n][e], rate, tail.softcap) : sc[n][e] * scale;
        if (bias && gid + 8 * r < heads) v += bias[(size_t)(h0 + gid + 8 * r) * reach + max(0, min(p - key, reach - 1))];
        if (!(kept ? key < keep_first : (key >= lo && key <= p))) v = -INFINITY;
        sc[n][e] = v;
        top[r] = fmaxf(top[r], v);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (r == 1 && heads <= 8) break;
      top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 1));
      top[r] = fmaxf(top[r], __shfl_xor_sync(0xffffffffu, top[r], 2));
      const float m_new = fmaxf(m[r], top[r]), alpha = expf(m[r] - m_new);
      m[r] = m_new;
      l[r] *= alpha;
#pragma unroll
      for (int i = 0; i < V / 8; ++i) { o[i][2 * r] *= alpha; o[i][2 * r + 1] *= alpha; }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (e >> 1 == 1 && heads <= 8) { sc[n][e] = 0.f; continue; }
        sc[n][e] = expf(sc[n][e] - m[e >> 1]);  // a masked score is -inf: weight 0
        l[e >> 1] += sc[n][e];
      }
    uint32_t hi[4], lo4[4];
    split_bf16(sc[0][0], sc[0][1], hi[0], lo4[0]);
    split_bf16(sc[0][2], sc[0][3], hi[1], lo4[1]);
    split_bf16(sc[1][0], sc[1][1], hi[2], lo4[2]);
    split_bf16(sc[1][2], sc[1][3], hi[3], lo4[3]);
#pragma unroll
    for (int nv = 0; nv < V / 8; nv += 2) {
      if (nv * 8 >= vdim) break;
      uint32_t b[4];  // (values in an odd number of eights: the last columns read 16 bytes beyond the row, and nobody stores them)
      rows_ldmatrix4_trans(b, src + (uint32_t)(((lmat & 1) * 8 + lrow) * pitch + dim + nv * 8 + (lmat >> 1) * 8) * 2);
      mma_16816(o[nv], hi[0], hi[1], hi[2], hi[3], b[0], b[1]);
      mma_16816(o[nv], lo4[0], lo4[1], lo4[2], lo4[3], b[0], b[1]);
      mma_16816(o[nv + 1], hi[0], hi[1], hi[2], hi[3], b[2], b[3]);
      mma_16816(o[nv + 1], lo4[0], lo4[1], lo4[2], lo4[3], b[2], b[3]);
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
  }
  __syncthreads();  // every warp has left its ring: the shares take its place, [warp][head][vdim | m | l]
  float* join = reinterpret_cast<float*>(rows_raw);
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = gid + 8 * r;
    if (row >= heads) continue;
    float* dst = join + ((size_t)warp * ROWS_HEADS + row) * (vdim + 2);
#pragma unroll
    for (int i = 0; i < V / 8; ++i) {
      const int c = i * 8 + 2 * tig;
      if (c < vdim) { dst[c] = o[i][2 * r]; dst[c + 1] = o[i][2 * r + 1]; }
    }
    if (tig == 0) { dst[vdim] = m[r]; dst[vdim + 1] = l[r]; }
  }
  __syncthreads();
  for (int row = warp; row < heads; row += ROWS_WARPS) {  // a warp a head
    const int h = h0 + row;
    const bool sink_here = sink && splits == 1;
    float M = sink_here ? sink[h] : -FLT_MAX;
    float mw[ROWS_WARPS], f[ROWS_WARPS];
#pragma unroll
    for (int w = 0; w < ROWS_WARPS; ++w) {
      mw[w] = join[((size_t)w * ROWS_HEADS + row) * (vdim + 2) + vdim];
      M = fmaxf(M, mw[w]);
    }
    float L = sink_here ? expf(sink[h] - M) : 0.f;
#pragma unroll
    for (int w = 0; w < ROWS_WARPS; ++w) {
      f[w] = expf(mw[w] - M);
      L += join[((size_t)w * ROWS_HEADS + row) * (vdim + 2) + vdim + 1] * f[w];
    }
    if (splits > 1) {
      float* dst = partial + (((size_t)t * hq + h) * splits + blockIdx.y) * (vdim + 2);
      if (lane == 0) { dst[0] = M; dst[1] = L; }
      for (int d = lane; d < vdim; d += 32) {
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < ROWS_WARPS; ++w) sum = fmaf(join[((size_t)w * ROWS_HEADS + row) * (vdim + 2) + d], f[w], sum);
        dst[2 + d] = sum;
      }
    } else {
      const float inv = 1.f / L;
      for (int d = lane; d < vdim; d += 32) {
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < ROWS_WARPS; ++w) sum = fmaf(join[((size_t)w * ROWS_HEADS + row) * (vdim + 2) + d], f[w], sum);
        out[(size_t)t * tail.ldo + (size_t)h * vdim + d] =
            __float2bfloat16_rn(sum * inv * tail_factor<__nv_bfloat16>(tail, t, h * vdim + d));
      }
    }
  }
}

size_t tile_smem(int dp, int vp, int share) {
  return sizeof(float) * ((size_t)dp * 33 + 32 * (size_t)vp + (size_t)TILE_T * share * dp + 2 * (size_t)TILE_T * share +
                          (size_t)TILE_T * share * vp);
}

PsbPerDevice tile_attr[4][4];

int padded(int n) { return n <= 32 ? 32 : n <= 64 ? 64 : n <= 128 ? 128 : 256; }
int slot_of(int n) { return n == 32 ? 0 : n == 64 ? 1 : n == 128 ? 2 : 3; }

}  // namespace

// (qkv, dtype, positions, token_item, table, table_width, kv, kv_dtype, q_out, T, hq, hkv, dim, vdim, page_size, num_pages, stream)
PSB_API int psb_attention_biased_append(const void* qkv, int dtype, const void* positions, const void* token_item,
                                        const void* table, int table_width, void* kv, int kv_dtype, void* q_out, int T, int hq,
                                        int hkv, int dim, int vdim, int page_size, int num_pages, cudaStream_t stream) {
  if (T < 0 || hq < 1 || hkv < 1 || dim < 1 || vdim < 1 || page_size < 1 || table_width < 1 || num_pages < 1)
    PSB_REFUSE("attention_biased_append: bad sizes");
  if (T == 0) return 0;
  PSB_DISPATCH_DTYPE(dtype, T_, {
    PSB_DISPATCH_DTYPE(kv_dtype, TKV, {
      psb_launch(attention_biased_append_kernel<T_, TKV>, dim3(T), dim3(128), 0, stream, (const T_*)qkv, (const int32_t*)positions,
                 (const int32_t*)token_item, (const int32_t*)table, table_width, (TKV*)kv, (T_*)q_out, hq, hkv, dim, vdim,
                 page_size, num_pages);
    });
  });
  PSB_LAUNCH_CHECK("attention_biased_append");
  return 0;
}

// ``skip_from`` > 0: tokens of portions with at least that many tokens are left to the tiled kernel (item_start needed).
// (q, dtype, kv, kv_dtype, table, table_width, positions, token_item, bias, sink, out, T, hq, hkv, dim, vdim, page_size,
//  window, chunk, reach, scale, item_start, skip_from, keep_first, partial [T * hq, splits, vdim + 2] float32 or null, splits,
//  gate, ldg, ldo, out_scale, softcap, stream); gate (or null) has the type of q
PSB_API int psb_attention_biased(const void* q, int dtype, const void* kv, int kv_dtype, const void* table, int table_width,
                                 const void* positions, const void* token_item, const void* bias, const void* sink, void* out,
                                 int T, int hq, int hkv, int dim, int vdim, int page_size, int window, int chunk, int reach,
                                 float scale, const void* item_start, int skip_from, int keep_first, void* partial, int splits,
                                 const void* gate, long long ldg, long long ldo, float out_scale, float softcap, cudaStream_t stream) {
  if (ldo < (long long)hq * vdim || (gate && ldg < (long long)hq * vdim) || softcap < 0.f) PSB_REFUSE("attention_biased: bad output or gate rows, or a negative cap");
  const RowsTail tail{gate, ldg, ldo, out_scale, softcap};
  if (splits < 1 || splits > MAX_KEY_SPLITS || (splits > 1 && (!partial || skip_from > 0)))
    PSB_REFUSE("attention_biased: 1 to %d shares of the keys (with their scratch, and no tokens left to another kernel), not %d", MAX_KEY_SPLITS, splits);
  if (keep_first < 0 || (keep_first > 0 && (window < 1 || chunk > 0))) PSB_REFUSE("attention_biased: kept first keys go with a window and no chunk mask");
  if (skip_from > 0 && !item_start) PSB_REFUSE("attention_biased: skipping tiled portions needs the item offsets");
  if (T < 0 || hq < 1 || hkv < 1 || hq % hkv) PSB_REFUSE("attention_biased: %d query heads cannot share %d key/value heads", hq, hkv);
  if (dim < 1 || dim > MAX_D || vdim < 1 || vdim > MAX_D) PSB_REFUSE("attention_biased: sizes %d/%d are outside [1, %d]", dim, vdim, MAX_D);
  if (page_size < 1 || table_width < 1) PSB_REFUSE("attention_biased: bad paging (page_size=%d width=%d)", page_size, table_width);
  if (window < 0 || chunk < 0 || (bias && reach < 1)) PSB_REFUSE("attention_biased: negative window or chunk, or an empty bias table");
  if (T == 0) return 0;
  const long long blocks = (long long)T * hq;
  if (blocks > 0x7fffffffLL) PSB_REFUSE("attention_biased: batch too large");
  PSB_DISPATCH_DTYPE(dtype, T_, {
    PSB_DISPATCH_DTYPE(kv_dtype, TKV, {
      psb_launch(attention_biased_kernel<T_, TKV>, dim3((unsigned)blocks, (unsigned)splits), dim3(WARPS * 32), 0, stream, (const T_*)q,
                 (const TKV*)kv, (const int32_t*)table, table_width, (const int32_t*)positions, (const int32_t*)token_item,
                 (const float*)bias, (const float*)sink, (T_*)out, T, hq, hkv, dim, vdim, page_size, window, chunk, reach, scale,
                 (const int32_t*)item_start, skip_from, keep_first, (float*)partial, splits, tail);
    });
  });
  PSB_LAUNCH_CHECK("attention_biased");
  if (splits > 1) {
    PSB_DISPATCH_DTYPE(dtype, T_, {
      psb_launch(attention_biased_merge_kernel<T_>, dim3((unsigned)blocks), dim3(32), 0, stream, (const float*)partial,
                 (const float*)sink, (T_*)out, hq, vdim, splits, tail);
    });
    PSB_LAUNCH_CHECK("attention_biased_merge");
  }
  return 0;
}

// (hq, hkv, dim, vdim) -> 1 if the tensor-core kernel for single tokens takes the shape
PSB_API int psb_attention_rows_single_supported(int hq, int hkv, int dim, int vdim) {
  return hq >= 1 && hkv >= 1 && hq % hkv == 0 && dim >= 8 && dim <= 128 && dim % 8 == 0 && vdim >= 8 && vdim <= 128 && vdim % 8 == 0 ? 1 : 0;
}

// Every token alone (bfloat16), arguments as for psb_attention_biased; no token is skipped.
// (q, kv, table, table_width, positions, token_item, bias, sink, out, T, hq, hkv, dim, vdim, page_size, window, chunk, reach, scale,
//  keep_first, partial [T * hq, splits, vdim + 2] float32 or null, splits, gate, ldg, ldo, out_scale, softcap, stream)
PSB_API int psb_attention_rows_single(const void* q, const void* kv, const void* table, int table_width, const void* positions,
                                      const void* token_item, const void* bias, const void* sink, void* out, int T, int hq, int hkv,
                                      int dim, int vdim, int page_size, int window, int chunk, int reach, float scale, int keep_first,
                                      void* partial, int splits, const void* gate, long long ldg, long long ldo, float out_scale,
                                      float softcap, cudaStream_t stream) {
  if (!psb_attention_rows_single_supported(hq, hkv, dim, vdim)) PSB_REFUSE("attention_rows_single: shape not taken");
  if (splits < 1 || splits > MAX_KEY_SPLITS || (splits > 1 && !partial)) PSB_REFUSE("attention_rows_single: 1 to %d shares of the keys (with their scratch), not %d", MAX_KEY_SPLITS, splits);
  if (keep_first < 0 || (keep_first > 0 && (window < 1 || chunk > 0))) PSB_REFUSE("attention_rows_single: kept first keys go with a window and no chunk mask");
  if (T < 0 || page_size < 1 || table_width < 1 || window < 0 || chunk < 0 || (bias && reach < 1)) PSB_REFUSE("attention_rows_single: bad arguments");
  if (ldo < (long long)hq * vdim || (gate && ldg < (long long)hq * vdim) || softcap < 0.f) PSB_REFUSE("attention_rows_single: bad output or gate rows, or a negative cap");
  if (((uintptr_t)kv & 15) || ((uintptr_t)q & 3)) PSB_REFUSE("attention_rows_single: cache rows must start on 16 bytes");
  if (T == 0) return 0;
  const RowsTail tail{gate, ldg, ldo, out_scale, softcap};
  const int groups = (hq / hkv + ROWS_HEADS - 1) / ROWS_HEADS;
  const long long blocks = (long long)T * hkv * groups;
  if (blocks > 0x7fffffffLL) PSB_REFUSE("attention_rows_single: batch too large");
  const size_t smem = rows_smem(dim, vdim);
#define ROWS_CASE(D_, V_)                                                                                                      \
  do {                                                                                                                         \
    static PsbPerDevice configured;                                                                                            \
    if (!configured.get()) {                                                                                                   \
      if (cudaFuncSetAttribute(attention_rows_single_kernel<D_, V_>, cudaFuncAttributeMaxDynamicSharedMemorySize,               \
                               (int)rows_smem(D_, V_)) != cudaSuccess)                                                         \
        PSB_REFUSE("attention_rows_single: cannot raise the shared-memory limit");                                             \
      configured.set();                                                                                                        \
    }                                                                                                                          \
    psb_launch(attention_rows_single_kernel<D_, V_>, dim3((unsigned)blocks, (unsigned)splits), dim3(ROWS_WARPS * 32), smem, stream, \
               (const __nv_bfloat16*)q, (const __nv_bfloat16*)kv, (const int32_t*)table, table_width, (const int32_t*)positions, \
               (const int32_t*)token_item, (const float*)bias, (const float*)sink, (__nv_bfloat16*)out, hq, hkv, dim, vdim,     \
               page_size, window, chunk, reach, scale, keep_first, (float*)partial, splits, tail);                             \
  } while (0)
  if (dim <= 64 && vdim <= 64) ROWS_CASE(64, 64);
  else if (dim <= 64) ROWS_CASE(64, 128);
  else if (vdim <= 64) ROWS_CASE(128, 64);
  else ROWS_CASE(128, 128);
#undef ROWS_CASE
  PSB_LAUNCH_CHECK("attention_rows_single");
  if (splits > 1) {
    psb_launch(attention_biased_merge_kernel<__nv_bfloat16>, dim3((unsigned)(T * hq)), dim3(32), 0, stream, (const float*)partial,
               (const float*)sink, (__nv_bfloat16*)out, hq, vdim, splits, tail);
    PSB_LAUNCH_CHECK("attention_biased_merge");
  }
  return 0;
}

// (hq, hkv, dim, vdim) -> 1 if the tensor-core kernel for prompt portions takes the shape
PSB_API int psb_attention_biased_mma_supported(int hq, int hkv, int dim, int vdim) {
  return hq >= 1 && hkv >= 1 && hq % hkv == 0 && dim >= 8 && dim <= 128 && dim % 8 == 0 && vdim >= 8 && vdim <= 128 && vdim % 8 == 0 ? 1 : 0;
}

// The tensor-core kernel over every portion of at least ``min_tokens`` tokens (bfloat16; grid sized by an upper bound on
// the tiles).  Other tokens are left untouched.
// (q, kv, table, table_width, positions, item_start, items, T, min_tokens, bias, sink, out, hq, hkv, dim, vdim,
//  page_size, window, chunk, reach, scale, keep_first, gate, ldg, ldo, out_scale, softcap, stream)
PSB_API int psb_attention_biased_mma(const void* q, const void* kv, const void* table, int table_width, const void* positions,
                                     const void* item_start, int items, int T, int min_tokens, const void* bias, const void* sink,
                                     void* out, int hq, int hkv, int dim, int vdim, int page_size, int window, int chunk, int reach,
                                     float scale, int keep_first, const void* gate, long long ldg, long long ldo, float out_scale,
                                     float softcap, cudaStream_t stream) {
  if (ldo < (long long)hq * vdim || ldo % 2 || ((uintptr_t)out & 3) || (gate && ldg < (long long)hq * vdim) || softcap < 0.f)
    PSB_REFUSE("attention_biased_mma: bad output or gate rows, or a negative cap");
  const RowsTail tail{gate, ldg, ldo, out_scale, softcap};
  if (!psb_attention_biased_mma_supported(hq, hkv, dim, vdim)) PSB_REFUSE("attention_biased_mma: shape not taken");
  if (keep_first < 0 || (keep_first > 0 && (window < 1 || chunk > 0))) PSB_REFUSE("attention_biased_mma: kept first keys go with a window and no chunk mask");
  if (page_size < 1 || table_width < 1 || window < 0 || chunk < 0 || (bias && reach < 1)) PSB_REFUSE("attention_biased_mma: bad arguments");
  if ((((uintptr_t)q | (uintptr_t)kv) & 15) || hq > 65535) PSB_REFUSE("attention_biased_mma: operands must be 16-byte aligned");
  if (items < 1 || T < 1 || min_tokens < 1) return 0;
  // two heads that read the same keys and values share a block (64 tokens each) where there are such heads
  const int heads_here = (hq / hkv) % 2 == 0 ? 2 : 1, tile_tokens = 16 * MMA_WARPS / heads_here;
  const int by_chunk = items == 1 && chunk >= 2 * tile_tokens ? chunk / tile_tokens : 0;  // tiles of a last chunk that is cut off
  const dim3 grid(hq / heads_here, (T + tile_tokens - 1) / tile_tokens + items + by_chunk);
  if (grid.y > 65535) PSB_REFUSE("attention_biased_mma: %d tokens are too many for one launch", T);
  const size_t smem = mma_smem(dim, vdim, bias != nullptr, heads_here);
#define MMA_CASE(D_, V_)                                                                                                       \
  do {                                                                                                                         \
    static PsbPerDevice configured;                                                                                            \
    if (!configured.get()) {                                                                                                   \
      if (cudaFuncSetAttribute(attention_biased_mma_kernel<D_, V_>, cudaFuncAttributeMaxDynamicSharedMemorySize,                \
                               (int)mma_smem(D_, V_, true, 2)) != cudaSuccess)                                                 \
        PSB_REFUSE("attention_biased_mma: cannot raise the shared-memory limit");                                              \
      configured.set();                                                                                                        \
    }                                                                                                                          \
    psb_launch(attention_biased_mma_kernel<D_, V_>, grid, dim3(MMA_WARPS * 32), smem, stream, (const __nv_bfloat16*)q,          \
               (const __nv_bfloat16*)kv, (const int32_t*)table, table_width, (const int32_t*)positions,                        \
               (const int32_t*)item_start, items, min_tokens, (const float*)bias, (const float*)sink, (__nv_bfloat16*)out, hq,  \
               hkv, dim, vdim, page_size, window, chunk, reach, scale, keep_first, heads_here, tail);                          \
  } while (0)
  if (dim <= 64 && vdim <= 64) MMA_CASE(64, 64);
  else if (dim <= 64) MMA_CASE(64, 128);
  else if (vdim <= 64) MMA_CASE(128, 64);
  else MMA_CASE(128, 128);
#undef MMA_CASE
  PSB_LAUNCH_CHECK("attention_biased_mma");
  return 0;
}

// () -> tokens a tile of the tiled kernel holds
PSB_API int psb_attention_biased_tile_tokens() { return TILE_T; }

// (hq, hkv, dim, vdim) -> 1 if the tiled kernel takes the shape
PSB_API int psb_attention_biased_tile_supported(int hq, int hkv, int dim, int vdim) {
  if (hq < 1 || hkv < 1 || hq % hkv || dim < 1 || dim > MAX_D || vdim < 1 || vdim > MAX_D) return 0;
  const int dp = padded(dim), vp = padded(vdim);
  return tile_smem(dp, vp, hq / hkv) <= 200 * 1024 ? 1 : 0;
}

// The tiled kernel over every portion of at least ``min_tokens`` tokens (the grid is sized by an upper bound on their
// tiles, so its shape depends on T and the number of items only).  Other tokens are left untouched.
// (q, kv, table, table_width, positions, item_start, items, T, min_tokens, bias, sink, out, hq, hkv, dim, vdim,
//  page_size, window, chunk, reach, scale, keep_first, gate, ldg, ldo, out_scale, softcap, stream)
PSB_API int psb_attention_biased_tiles(const void* q, const void* kv, const void* table, int table_width, const void* positions,
                                       const void* item_start, int items, int T, int min_tokens,
                                       const void* bias, const void* sink, void* out, int hq, int hkv, int dim, int vdim,
                                       int page_size, int window, int chunk, int reach, float scale, int keep_first,
                                       const void* gate, long long ldg, long long ldo, float out_scale, float softcap,
                                       cudaStream_t stream) {
  if (ldo < (long long)hq * vdim || (gate && ldg < (long long)hq * vdim) || softcap < 0.f) PSB_REFUSE("attention_biased_tiles: bad output or gate rows, or a negative cap");
  const RowsTail tail{gate, ldg, ldo, out_scale, softcap};
  if (keep_first < 0 || (keep_first > 0 && (window < 1 || chunk > 0))) PSB_REFUSE("attention_biased_tiles: kept first keys go with a window and no chunk mask");
  if (items < 1 || T < 1 || min_tokens < 1) return 0;
  const int tiles = (T + TILE_T - 1) / TILE_T + items;
  if (!psb_attention_biased_tile_supported(hq, hkv, dim, vdim)) PSB_REFUSE("attention_biased_tiles: shape not taken");
  if (page_size < 1 || table_width < 1 || window < 0 || chunk < 0 || (bias && reach < 1)) PSB_REFUSE("attention_biased_tiles: bad arguments");
  if (hkv > 65535) PSB_REFUSE("attention_biased_tiles: too many key/value heads");
  const int dp = padded(dim), vp = padded(vdim);
  const size_t smem = tile_smem(dp, vp, hq / hkv);
  const dim3 grid(tiles, hkv), block(TILE_WARPS * 32);
#define TILE_CASE(DP_, VP_)                                                                                                    \
  if (dp == DP_ && vp == VP_) {                                                                                                \
    auto kernel = attention_biased_tile_kernel<DP_, VP_>;                                                                      \
    PsbPerDevice& done = tile_attr[slot_of(DP_)][slot_of(VP_)];                                                                \
    if (!done.get()) {                                                                                                         \
      if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)                \
        PSB_REFUSE("attention_biased_tiles: cannot raise the shared-memory limit");                                            \
      done.set();                                                                                                              \
    }                                                                                                                          \
    psb_launch(kernel, grid, block, smem, stream, (const __nv_bfloat16*)q, (const __nv_bfloat16*)kv, (const int32_t*)table,    \
               table_width, (const int32_t*)positions, (const int32_t*)item_start, items, min_tokens,                          \
               (const float*)bias, (const float*)sink, (__nv_bfloat16*)out, hq, hkv, dim, vdim,                                \
               page_size, window, chunk, reach, scale, keep_first, tail);                                                      \
    launched = true;                                                                                                           \
  }
#define TILE_ROW(DP_) TILE_CASE(DP_, 32) TILE_CASE(DP_, 64) TILE_CASE(DP_, 128) TILE_CASE(DP_, 256)
  bool launched = false;
  TILE_ROW(32) TILE_ROW(64) TILE_ROW(128) TILE_ROW(256)
#undef TILE_ROW
#undef TILE_CASE
  if (!launched) PSB_REFUSE("attention_biased_tiles: sizes %d/%d not instantiated", dim, vdim);
  PSB_LAUNCH_CHECK("attention_biased_tiles");
  return 0;
}

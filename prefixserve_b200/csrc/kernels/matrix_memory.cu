// Matrix memory with exponential gates: per request and head a state S [dim, vdim], a normalizer n [dim] and the exponent m they
// are divided by (both hold their true value times exp(-m)), all float32, from zero.  A token brings a log input gate
// i = cap tanh(z_i / cap) and a log forget gate f = logsigmoid(cap tanh(z_f / cap)):
//
//   m' = max(f + m, i),  S <- exp(f + m - m') S + exp(i - m') k v^T,  n <- exp(f + m - m') n + exp(i - m') k,
//   o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)            with q times dim^-1/2.
//
// The read-out of a head is divided by its root mean square over vdim, multiplied by a gain per head and channel and by the
// sigmoid of an output gate, and rounded to the compute type.  Everything is read where the layer's input product left it:
// rows ``ld`` numbers apart, [q: H dim | k: H dim | v: H vdim | gate: H vdim | z_i: H | z_f: H].
//
// A request's slot holds [S: H dim vdim | n: H NB dim | m: H NB]; NB = ceil(vdim / columns a block of the first kernel works on):
// every block keeps its own copy of n and m, so none waits for another.
//
// matrix_memory_step_kernel (any sizes, float32 and bfloat16): a block per request, head and run of columns goes through the
// portion token by token with the state in registers (R lanes hold the rows, four columns a lane).  One column block a head
// (NB = 1): norm, gain and gate ride along; else the read-out goes to a float32 tensor and normed_readout finishes it.
//
// Long bfloat16 portions are cut into chunks of 64 tokens that run side by side, on the tensor cores.  With F the running sum of
// f from a chunk's start, G = i - F and m_in the exponent at the chunk's start, m_t = F_t + max(m_in, max_(j <= t) G_j):
//   matrix_memory_chunk_kernel   every chunk from a zero state: sum_j exp(G_j - max G) k_j v_j^T, the same with k alone, F and
//                                F + max G at its end;
//   matrix_memory_starts_kernel  chunk by chunk: the state every chunk starts from, and what the slot holds afterwards;
//   matrix_memory_read_kernel    exp(F_i + G_j - m_i) (q_i . k_j) over the chunk's own tokens j <= i, times v_j, plus
//                                exp(F_i + m_in - m_i) q_i^T S; the normalizer likewise; norm, gain and gate.
// Factors that carry a float32 number enter a product as the sum of two bfloat16 numbers (16 bits); sums are float32.
#include "common.cuh"

namespace {

constexpr float READOUT_EPS = 1e-6f;
constexpr int MM_CHUNK = 64;    // tokens a chunk

__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) {
  const float x = cap * tanhf(z / cap);
  return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}

template <typename T>
struct MemoryArgs {
  const T* proj;
  long long ld;
  const float *bias_i, *bias_f;   // [H]
  const float* gain;              // [H, vdim]
  float* state;
  long long slot_floats;
  const int32_t *item_start, *slots;
  T* out;                         // rows ldo numbers apart: the finished read-out (NB == 1)
  long long ldo;
  float* o32;                     // [T, H, vdim]: the bare read-out (NB > 1)
  int items, H, dim, vdim, nb, num_slots;
  float cap, eps, scale;
};

template <typename T>
__device__ __forceinline__ float* slot_state(const MemoryArgs<T>& a, int item) {
  int slot = a.slots[item];
  slot = slot < 0 ? 0 : (slot >= a.num_slots ? a.num_slots - 1 : slot);
  return a.state + (size_t)slot * a.slot_floats;
}

// ---- token by token ---------------------------------------------------------------------------------------------

// A lane's rows of S: runs of four, 4 R apart.
template <int R>
__device__ __forceinline__ int row_of(int r, int e) { return (e >> 2) * (4 * R) + r * 4 + (e & 3); }

// Tokens the step kernel stages at a time.
constexpr int stage_tokens(int rows) { return rows <= 512 ? 8 : 4; }

template <typename T, int PER, int R, int WARPS>
__global__ void __launch_bounds__(WARPS * 32)
matrix_memory_step_kernel(const MemoryArgs<T> a) {
  constexpr int QUADS = 32 / R, COLS = 4 * QUADS, RP = PER * R, BC = WARPS * COLS, STAGE = stage_tokens(RP);
  __shared__ __align__(16) float qs[STAGE][RP], ks[STAGE][RP], vs[STAGE][BC];
  __shared__ float gi[STAGE], gf[STAGE];
  extern __shared__ float os[];  // [STAGE][BC]: the stage's read-outs (NB == 1)
  pdl_trigger();
  pdl_wait();
  const int item = blockIdx.z, h = blockIdx.y, cb = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane % R;
  const int t0 = a.item_start[item], t1 = a.item_start[item + 1];
  if (t0 >= t1) return;
  const int dim = a.dim, vdim = a.vdim, H = a.H;
  const int in_block = warp * COLS + lane / R * 4, col = cb * BC + in_block;
  float* slot = slot_state(a, item);
  float* S = slot + (size_t)h * dim * vdim;
  float* N = slot + (size_t)H * dim * vdim + ((size_t)h * a.nb + cb) * dim;
  float* M = slot + (size_t)H * dim * (vdim + a.nb) + (size_t)h * a.nb + cb;
  const bool quad = vdim % 4 == 0 && (((uintptr_t)S) & 15) == 0;
  const int warps = blockDim.x >> 5;  // narrow heads launch fewer warps

  float s[PER][4], n[PER];
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int d = row_of<R>(r, e);
    n[e] = d < dim ? N[d] : 0.f;
    s[e][0] = s[e][1] = s[e][2] = s[e][3] = 0.f;
    if (d >= dim) continue;
    if (quad) {
      if (col < vdim) {
        const float4 v = *reinterpret_cast<const float4*>(S + (size_t)d * vdim + col);
        s[e][0] = v.x; s[e][1] = v.y; s[e][2] = v.z; s[e][3] = v.w;
      }
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (col + j < vdim) s[e][j] = S[(size_t)d * vdim + col + j];
    }
  }
  float m = *M;
  const T* qsrc = a.proj + (size_t)h * dim;
  const T* ksrc = qsrc + (size_t)H * dim;
  const T* vsrc = a.proj + 2 * (size_t)H * dim + (size_t)h * vdim;
  const T* gsrc = vsrc + (size_t)H * vdim;
  const T* zsrc = a.proj + 2 * (size_t)H * (dim + vdim) + h;
  const int cols_here = min(BC, vdim - cb * BC);

  for (int ts = t0; ts < t1; ts += STAGE) {
    const int live = min(STAGE, t1 - ts);
    __syncthreads();  // everybody is done with the stage before
    for (int i = threadIdx.x; i < live * RP; i += blockDim.x) {
      const int tok = i / RP, d = i - tok * RP;
      const size_t row = (size_t)(ts + tok) * a.ld;
      qs[tok][d] = d < dim ? to_float<T>(qsrc[row + d]) * a.scale : 0.f;
      ks[tok][d] = d < dim ? to_float<T>(ksrc[row + d]) : 0.f;
    }
    for (int i = threadIdx.x; i < live * BC; i += blockDim.x) {
      const int tok = i / BC, c = i - tok * BC;
      vs[tok][c] = c < cols_here ? to_float<T>(vsrc[(size_t)(ts + tok) * a.ld + cb * BC + c]) : 0.f;
    }
    if (threadIdx.x < live) {
      const T* z = zsrc + (size_t)(ts + threadIdx.x) * a.ld;
      gi[threadIdx.x] = log_input_gate(to_float<T>(z[0]) + a.bias_i[h], a.cap);
      gf[threadIdx.x] = log_forget_gate(to_float<T>(z[H]) + a.bias_f[h], a.cap);
    }
    __syncthreads();
#pragma unroll 1
    for (int i = 0; i < live; ++i) {
      const float top = fmaxf(gf[i] + m, gi[i]);
      const float keep = expf(gf[i] + m - top), write = expf(gi[i] - top);
      m = top;
      const float4 v4 = *reinterpret_cast<const float4*>(&vs[i][in_block]);
      const float v[4] = {v4.x, v4.y, v4.z, v4.w};
      float o[4] = {}, den = 0.f;
#pragma unroll
      for (int e = 0; e < PER; e += 4) {
        const float4 k4 = *reinterpret_cast<const float4*>(&ks[i][row_of<R>(r, e)]);
        const float4 q4 = *reinterpret_cast<const float4*>(&qs[i][row_of<R>(r, e)]);
        const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float kw = write * kk[u];
          n[e + u] = fmaf(keep, n[e + u], kw);
          den = fmaf(n[e + u], qq[u], den);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            s[e + u][j] = fmaf(keep, s[e + u][j], kw * v[j]);
            o[j] = fmaf(s[e + u][j], qq[u], o[j]);
          }
        }
      }
      // sums over the R lanes: the first two rounds halve the columns a lane still sums
#pragma unroll
      for (int off = 1; off < R; off <<= 1) den += __shfl_xor_sync(0xffffffffu, den, off);
      int mine = 0;
#pragma unroll
      for (int w = 4, off = 1; w > 1; w >>= 1, off <<= 1) {
        const bool up = r & off;
#pragma unroll
        for (int j = 0; j < w / 2; ++j) {
          const float give = up ? o[j] : o[j + w / 2], hold = up ? o[j + w / 2] : o[j];
          o[j] = hold + __shfl_xor_sync(0xffffffffu, give, off);
        }
        mine += up ? w / 2 : 0;
      }
#pragma unroll
      for (int off = 4; off < R; off <<= 1) o[0] += __shfl_xor_sync(0xffffffffu, o[0], off);
      if (r < 4) {
        const float value = o[0] / (fmaxf(fabsf(den), expf(-m)) + READOUT_EPS);
        if (a.nb == 1) os[i * BC + in_block + mine] = value;
        else if (col + mine < vdim) a.o32[((size_t)(ts + i) * H + h) * vdim + col + mine] = value;
      }
    }
    if (a.nb == 1) {
      __syncthreads();
      for (int i = warp; i < live; i += warps) {  // a warp a token
        float ss = 0.f;
        for (int c = lane; c < vdim; c += 32) ss = fmaf(os[i * BC + c], os[i * BC + c], ss);
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)vdim + a.eps);
        const T* g = gsrc + (size_t)(ts + i) * a.ld;
        T* dst = a.out + (size_t)(ts + i) * a.ldo + (size_t)h * vdim;
        for (int c = lane; c < vdim; c += 32)
          dst[c] = from_float<T>(os[i * BC + c] * inv * a.gain[(size_t)h * vdim + c] / (1.f + expf(-to_float<T>(g[c]))));
      }
    }
  }
#pragma unroll
  for (int e = 0; e < PER; ++e) {
    const int d = row_of<R>(r, e);
    if (d >= dim) continue;
    if (warp == 0 && lane < R) N[d] = n[e];
    if (quad) {
      if (col < vdim) *reinterpret_cast<float4*>(S + (size_t)d * vdim + col) = make_float4(s[e][0], s[e][1], s[e][2], s[e][3]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (col + j < vdim) S[(size_t)d * vdim + col + j] = s[e][j];
    }
  }
  if (threadIdx.x == 0) *M = m;
}

// ---- chunks side by side --------------------------------------------------------------------------------------------

__device__ __forceinline__ void mma_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix4(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void ldmatrix4_trans(uint32_t (&r)[4], const __nv_bfloat16* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ uint32_t pack_bf16(float x, float y) {
  __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
  return *reinterpret_cast<uint32_t*>(&v);
}
// two numbers as the sums hi + lo of two bfloat16 each
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat16 hx = __float2bfloat16_rn(x), hy = __float2bfloat16_rn(y);
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - __bfloat162float(hx), y - __bfloat162float(hy));
}

// The chunk a block works on: chunks are numbered through the step's items in order.  False beyond the last.
__device__ __forceinline__ bool find_chunk(const int32_t* __restrict__ item_start, int items, int at, int& item, int& t0, int& t1) {
  for (int i = 0; i < items; ++i) {
    const int s = item_start[i], e = item_start[i + 1], n = (e - s + MM_CHUNK - 1) / MM_CHUNK;
    if (at < n) {
      item = i;
      t0 = s + at * MM_CHUNK;
      t1 = min(e, t0 + MM_CHUNK);
      return true;
    }
    at -= n;
  }
  return false;
}

// One warp: F[t] = f_1 + .. + f_t, G[t] = i_t - F[t], P[t] = max(G_1 .. G_t) of a chunk's tokens (tokens beyond its end write
// nothing: G = -inf).
__device__ __forceinline__ void chunk_gates(const MemoryArgs<__nv_bfloat16>& a, int h, int t0, int live, float* F, float* G, float* P) {
  const int lane = threadIdx.x & 31;
  const __nv_bfloat16* z = a.proj + 2 * (size_t)a.H * (a.dim + a.vdim) + h;
  float f[2], g[2];
#pragma unroll
  for (int u = 0; u < 2; ++u) {  // a lane holds two neighbouring tokens
    const int t = 2 * lane + u;
    f[u] = 0.f;
    g[u] = -INFINITY;
    if (t < live) {
      const __nv_bfloat16* row = z + (size_t)(t0 + t) * a.ld;
      g[u] = log_input_gate(__bfloat162float(row[0]) + a.bias_i[h], a.cap);
      f[u] = log_forget_gate(__bfloat162float(row[a.H]) + a.bias_f[h], a.cap);
    }
  }
  float before = f[0] + f[1];
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float x = __shfl_up_sync(0xffffffffu, before, o);
    if (lane >= o) before += x;
  }
  before -= f[0] + f[1];  // the sum in front of this lane's tokens
  const float F0 = before + f[0], F1 = F0 + f[1];
  g[0] -= F0;
  g[1] -= F1;
  float top = fmaxf(g[0], g[1]);
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float x = __shfl_up_sync(0xffffffffu, top, o);
    if (lane >= o) top = fmaxf(top, x);
  }
  float ahead = __shfl_up_sync(0xffffffffu, top, 1);
  if (lane == 0) ahead = -INFINITY;
  F[2 * lane] = F0; F[2 * lane + 1] = F1;
  G[2 * lane] = g[0]; G[2 * lane + 1] = g[1];
  P[2 * lane] = fmaxf(ahead, g[0]); P[2 * lane + 1] = top;
}

// rows [0, live) of ``width`` numbers from global memory into a tile of ``pitch`` columns, the rest zeros; 16 bytes a piece
__device__ __forceinline__ void load_tile(__nv_bfloat16* tile, int pitch, int padded, const __nv_bfloat16* src, long long ld, int live, int width) {
  const int pieces = padded / 8;
  for (int i = threadIdx.x; i < MM_CHUNK * pieces; i += blockDim.x) {
    const int t = i / pieces, c = (i - t * pieces) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (t < live && c < width) v = *reinterpret_cast<const uint4*>(src + (size_t)t * ld + c);
    *reinterpret_cast<uint4*>(tile + t * pitch + c) = v;
  }
}

constexpr int MM_THREADS = 256;

template <int D, int V>
struct ChunkShape {
  static constexpr int KP = D + 8, VP = V + 8;  // row pitches that keep ldmatrix off its own banks
  static constexpr int CHUNK_SMEM = MM_CHUNK * (KP + 2 * VP) * 2;
  static constexpr int SLAB = 64;               // rows of S a round of the read-out kernel holds
  static constexpr int READ_SMEM = (MM_CHUNK * (2 * KP + VP) + 2 * SLAB * VP) * 2;
};

// grid: (column blocks, H, chunks).  local_s [chunks, H, dim, vdim], local_n [chunks, H, dim], ends [chunks, H, 2] = F and
// F + max G at the chunk's end.
template <int D, int V>
__global__ void __launch_bounds__(MM_THREADS)
matrix_memory_chunk_kernel(const MemoryArgs<__nv_bfloat16> a, float* __restrict__ local_s, float* __restrict__ local_n,
                           float* __restrict__ ends) {
  using Z = ChunkShape<D, V>;
  constexpr int WM = D / 16 < 8 ? D / 16 : 8, WN = 8 / WM, MT = D / 16 / WM, NT = V / WN / 8;
  extern __shared__ __align__(16) __nv_bfloat16 tiles[];
  __nv_bfloat16 *kt = tiles, *vh = kt + MM_CHUNK * Z::KP, *vl = vh + MM_CHUNK * Z::VP;
  __shared__ float F[MM_CHUNK], G[MM_CHUNK], P[MM_CHUNK], weight[MM_CHUNK];
  pdl_trigger();
  pdl_wait();
  int item, t0, t1;
  if (!find_chunk(a.item_start, a.items, blockIdx.z, item, t0, t1)) return;
  const int h = blockIdx.y, c0 = blockIdx.x * V, live = t1 - t0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const __nv_bfloat16* row0 = a.proj + (size_t)t0 * a.ld;
  load_tile(kt, Z::KP, D, row0 + (size_t)(a.H + h) * a.dim, a.ld, live, a.dim);
  if (warp == 0) chunk_gates(a, h, t0, live, F, G, P);
  __syncthreads();
  const float top = P[MM_CHUNK - 1];
  if (threadIdx.x < MM_CHUNK) weight[threadIdx.x] = expf(G[threadIdx.x] - top);
  __syncthreads();
  // values times exp(G - max G), as two bfloat16 tiles
  for (int i = threadIdx.x; i < MM_CHUNK * (V / 8); i += MM_THREADS) {
    const int t = i / (V / 8), c = (i - t * (V / 8)) * 8;
    uint4 hi = make_uint4(0, 0, 0, 0), lo = hi;
    if (t < live && c0 + c < a.vdim) {
      const uint4 raw = *reinterpret_cast<const uint4*>(row0 + (size_t)t * a.ld + 2 * (size_t)a.H * a.dim + (size_t)h * a.vdim + c0 + c);
      const __nv_bfloat162* v2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
      const float w = weight[t];
      uint32_t *hp = reinterpret_cast<uint32_t*>(&hi), *lp = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 v = __bfloat1622float2(v2[j]);
        split_bf16(v.x * w, v.y * w, hp[j], lp[j]);
      }
    }
    *reinterpret_cast<uint4*>(vh + t * Z::VP + c) = hi;
    *reinterpret_cast<uint4*>(vl + t * Z::VP + c) = lo;
  }
  __syncthreads();
  const int wm = warp % WM, wn = warp / WM;
  const int g = lane >> 2, q = lane & 3, lrow = lane & 7, lmat = lane >> 3;
  float acc[MT][NT][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < MM_CHUNK; kk += 16) {
    uint32_t af[MT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)  // K^T: rows of the tile are tokens, the product's rows are channels
      ldmatrix4_trans(af[i], kt + (kk + (lmat >> 1) * 8 + lrow) * Z::KP + (i * WM + wm) * 16 + (lmat & 1) * 8);
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      uint32_t bh[4], bl[4];
      const int at = (kk + (lmat & 1) * 8 + lrow) * Z::VP + wn * (V / WN) + j * 8 + (lmat >> 1) * 8;
      ldmatrix4_trans(bh, vh + at);
      ldmatrix4_trans(bl, vl + at);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        mma_16816(acc[i][j], af[i], bh[0], bh[1]);
        mma_16816(acc[i][j], af[i], bl[0], bl[1]);
        mma_16816(acc[i][j + 1], af[i], bh[2], bh[3]);
        mma_16816(acc[i][j + 1], af[i], bl[2], bl[3]);
      }
    }
  }
  float* S = local_s + ((size_t)blockIdx.z * a.H + h) * a.dim * a.vdim;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int d = (i * WM + wm) * 16 + g, c = c0 + wn * (V / WN) + j * 8 + 2 * q;
      if (c >= a.vdim) continue;
      if (d < a.dim) *reinterpret_cast<float2*>(S + (size_t)d * a.vdim + c) = make_float2(acc[i][j][0], acc[i][j][1]);
      if (d + 8 < a.dim) *reinterpret_cast<float2*>(S + (size_t)(d + 8) * a.vdim + c) = make_float2(acc[i][j][2], acc[i][j][3]);
    }
  if (blockIdx.x == 0) {
    for (int d = threadIdx.x; d < a.dim; d += MM_THREADS) {
      float sum = 0.f;
      for (int t = 0; t < live; ++t) sum = fmaf(weight[t], __bfloat162float(kt[t * Z::KP + d]), sum);
      local_n[((size_t)blockIdx.z * a.H + h) * a.dim + d] = sum;
    }
    if (threadIdx.x == 0) {
      float* e = ends + ((size_t)blockIdx.z * a.H + h) * 2;
      e[0] = F[live - 1];
      e[1] = F[live - 1] + top;
    }
  }
}

// A thread per four numbers of a portion's S, then per number of its n: what every chunk brought becomes what it starts from
// (``starts`` [chunks, H]: the exponents), and the slot receives the portion's end.
__global__ void __launch_bounds__(256)
matrix_memory_starts_kernel(const MemoryArgs<__nv_bfloat16> a, float* __restrict__ local_s, float* __restrict__ local_n,
                            const float* __restrict__ ends, float* __restrict__ starts) {
  pdl_trigger();
  pdl_wait();
  const int item = blockIdx.y;
  int first = 0;
  for (int i = 0; i < item; ++i) first += (a.item_start[i + 1] - a.item_start[i] + MM_CHUNK - 1) / MM_CHUNK;
  const int n = (a.item_start[item + 1] - a.item_start[item] + MM_CHUNK - 1) / MM_CHUNK;
  const int per_head = a.dim * a.vdim, quads = a.H * (per_head / 4);
  const int at = blockIdx.x * blockDim.x + threadIdx.x;
  if (n < 1 || at >= quads + a.H * a.dim) return;
  float* slot = slot_state(a, item);
  float* held_n = slot + (size_t)a.H * per_head;
  float* held_m = held_n + (size_t)a.H * a.nb * a.dim;
  constexpr int AHEAD = 8;
  if (at < quads) {
    const int h = at / (per_head / 4);
    float4 run = reinterpret_cast<const float4*>(slot)[at];
    float m = held_m[(size_t)h * a.nb];
    float4* src = reinterpret_cast<float4*>(local_s) + (size_t)first * quads + at;
    for (int c0 = 0; c0 < n; c0 += AHEAD) {
      float4 b[AHEAD];
      float2 e[AHEAD];
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        const bool there = c0 + j < n;
        b[j] = there ? src[(size_t)(c0 + j) * quads] : make_float4(0.f, 0.f, 0.f, 0.f);
        e[j] = there ? *reinterpret_cast<const float2*>(ends + ((size_t)(first + c0 + j) * a.H + h) * 2) : make_float2(0.f, 0.f);
      }
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        if (c0 + j >= n) break;
        src[(size_t)(c0 + j) * quads] = run;
        const float top = fmaxf(e[j].x + m, e[j].y), keep = expf(e[j].x + m - top), add = expf(e[j].y - top);
        m = top;
        run.x = fmaf(keep, run.x, add * b[j].x);
        run.y = fmaf(keep, run.y, add * b[j].y);
        run.z = fmaf(keep, run.z, add * b[j].z);
        run.w = fmaf(keep, run.w, add * b[j].w);
      }
    }
    reinterpret_cast<float4*>(slot)[at] = run;
    return;
  }
  // the first thread of a head's n also leaves the exponents; m is read by threads of other blocks too, so the slot's m is
  // brought up to date by the read-out kernel, which starts after this one
  const int hd = at - quads, h = hd / a.dim, d = hd - h * a.dim;
  float run = held_n[(size_t)h * a.nb * a.dim + d];
  float m = held_m[(size_t)h * a.nb];
  for (int c = 0; c < n; ++c) {
    float* b = local_n + ((size_t)(first + c) * a.H + h) * a.dim + d;
    const float* e = ends + ((size_t)(first + c) * a.H + h) * 2;
    const float got = *b;
    *b = run;
    if (d == 0) starts[(size_t)(first + c) * a.H + h] = m;
    const float top = fmaxf(e[0] + m, e[1]);
    run = fmaf(expf(e[0] + m - top), run, expf(e[1] - top) * got);
    m = top;
  }
  for (int k = 0; k < a.nb; ++k) held_n[((size_t)h * a.nb + k) * a.dim + d] = run;
}

// grid: (column blocks, H, chunks); four warps along the chunk's tokens, two along the columns.
template <int D, int V>
__global__ void __launch_bounds__(MM_THREADS)
matrix_memory_read_kernel(const MemoryArgs<__nv_bfloat16> a, const float* __restrict__ start_s, const float* __restrict__ start_n,
                          const float* __restrict__ starts) {
  using Z = ChunkShape<D, V>;
  constexpr int NT = V / 2 / 8;  // tiles of eight columns a warp
  extern __shared__ __align__(16) __nv_bfloat16 tiles[];
  __nv_bfloat16 *qt = tiles, *kt = qt + MM_CHUNK * Z::KP, *vt = kt + MM_CHUNK * Z::KP, *sh = vt + MM_CHUNK * Z::VP, *sl = sh + Z::SLAB * Z::VP;
  __shared__ float F[MM_CHUNK], G[MM_CHUNK], P[MM_CHUNK], qn[MM_CHUNK], square[2][MM_CHUNK];
  pdl_trigger();
  pdl_wait();
  int item, t0, t1;
  if (!find_chunk(a.item_start, a.items, blockIdx.z, item, t0, t1)) return;
  const int h = blockIdx.y, c0 = blockIdx.x * V, live = t1 - t0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const __nv_bfloat16* row0 = a.proj + (size_t)t0 * a.ld;
  const size_t ch = (size_t)blockIdx.z * a.H + h;
  load_tile(qt, Z::KP, D, row0 + (size_t)h * a.dim, a.ld, live, a.dim);
  load_tile(kt, Z::KP, D, row0 + (size_t)(a.H + h) * a.dim, a.ld, live, a.dim);
  load_tile(vt, Z::VP, V, row0 + 2 * (size_t)a.H * a.dim + (size_t)h * a.vdim + c0, a.ld, live, min(V, a.vdim - c0));
  if (warp == 0) chunk_gates(a, h, t0, live, F, G, P);
  __syncthreads();
  const float m_in = starts[ch];
  {  // q . n of the chunk's start, four threads a token
    const int t = threadIdx.x >> 2;
    float sum = 0.f;
    for (int d = threadIdx.x & 3; d < a.dim; d += 4) sum = fmaf(__bfloat162float(qt[t * Z::KP + d]), start_n[ch * a.dim + d], sum);
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    if ((threadIdx.x & 3) == 0) qn[t] = sum;
  }
  const int wm = warp & 3, wn = warp >> 2;
  const int g = lane >> 2, q = lane & 3, lrow = lane & 7, lmat = lane >> 3;
  float acc[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;

  // q^T S of the chunk's start, SLAB rows of S at a time
  for (int d0 = 0; d0 < a.dim; d0 += Z::SLAB) {
    __syncthreads();
    for (int i = threadIdx.x; i < Z::SLAB * (V / 4); i += MM_THREADS) {
      const int r = i / (V / 4), c = (i - r * (V / 4)) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (d0 + r < a.dim && c0 + c < a.vdim) v = *reinterpret_cast<const float4*>(start_s + (ch * a.dim + d0 + r) * a.vdim + c0 + c);
      uint2 hi, lo;
      split_bf16(v.x, v.y, hi.x, lo.x);
      split_bf16(v.z, v.w, hi.y, lo.y);
      *reinterpret_cast<uint2*>(sh + r * Z::VP + c) = hi;
      *reinterpret_cast<uint2*>(sl + r * Z::VP + c) = lo;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < Z::SLAB; kk += 16) {
      uint32_t af[4];
      ldmatrix4(af, qt + (wm * 16 + (lmat & 1) * 8 + lrow) * Z::KP + d0 + kk + (lmat >> 1) * 8);
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        uint32_t bh[4], bl[4];
        const int at = (kk + (lmat & 1) * 8 + lrow) * Z::VP + wn * (V / 2) + j * 8 + (lmat >> 1) * 8;
        ldmatrix4_trans(bh, sh + at);
        ldmatrix4_trans(bl, sl + at);
        mma_16816(acc[j], af, bh[0], bh[1]);
        mma_16816(acc[j], af, bl[0], bl[1]);
        mma_16816(acc[j + 1], af, bh[2], bh[3]);
        mma_16816(acc[j + 1], af, bl[2], bl[3]);
      }
    }
  }
  // this thread's two tokens
  float shift[2], den[2], floor_[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = wm * 16 + g + 8 * r;
    const float m = F[t] + fmaxf(m_in, P[t]);
    const float carry = expf(F[t] + m_in - m) * a.scale;
    shift[r] = F[t] - m;
    floor_[r] = expf(-m);
    den[r] = q == 0 ? carry * qn[t] : 0.f;
#pragma unroll
    for (int j = 0; j < NT; ++j) { acc[j][2 * r] *= carry; acc[j][2 * r + 1] *= carry; }
  }
  // the chunk's own tokens, 16 keys at a time; both column halves work out the same weights
#pragma unroll 1
  for (int k0 = 0; k0 <= wm * 16; k0 += 16) {
    float sc[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < D; kk += 16) {
      uint32_t af[4], bf[4];
      ldmatrix4(af, qt + (wm * 16 + (lmat & 1) * 8 + lrow) * Z::KP + kk + (lmat >> 1) * 8);
      ldmatrix4(bf, kt + (k0 + (lmat >> 1) * 8 + lrow) * Z::KP + kk + (lmat & 1) * 8);
      mma_16816(sc[0], af, bf[0], bf[1]);
      mma_16816(sc[1], af, bf[2], bf[3]);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = e >> 1, key = k0 + n * 8 + 2 * q + (e & 1);
        const float w = key <= wm * 16 + g + 8 * r ? sc[n][e] * a.scale * expf(shift[r] + G[key]) : 0.f;
        sc[n][e] = w;
        den[r] += w;
      }
    uint32_t hi[4], lo[4];
    split_bf16(sc[0][0], sc[0][1], hi[0], lo[0]);
    split_bf16(sc[0][2], sc[0][3], hi[1], lo[1]);
    split_bf16(sc[1][0], sc[1][1], hi[2], lo[2]);
    split_bf16(sc[1][2], sc[1][3], hi[3], lo[3]);
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      uint32_t bv[4];
      ldmatrix4_trans(bv, vt + (k0 + (lmat & 1) * 8 + lrow) * Z::VP + wn * (V / 2) + j * 8 + (lmat >> 1) * 8);
      mma_16816(acc[j], hi, bv[0], bv[1]);
      mma_16816(acc[j], lo, bv[0], bv[1]);
      mma_16816(acc[j + 1], hi, bv[2], bv[3]);
      mma_16816(acc[j + 1], lo, bv[2], bv[3]);
    }
  }
  float inv[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    den[r] += __shfl_xor_sync(0xffffffffu, den[r], 1);
    den[r] += __shfl_xor_sync(0xffffffffu, den[r], 2);
    inv[r] = 1.f / (fmaxf(fabsf(den[r]), floor_[r]) + READOUT_EPS);
  }
  if (t1 == a.item_start[item + 1] && blockIdx.x == 0 && threadIdx.x == 0) {  // the portion's last chunk leaves its exponent
    float* held_m = slot_state(a, item) + (size_t)a.H * a.dim * (a.vdim + a.nb) + (size_t)h * a.nb;
    const float m = F[live - 1] + fmaxf(m_in, P[live - 1]);
    for (int k = 0; k < a.nb; ++k) held_m[k] = m;
  }
  if (a.nb > 1) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = wm * 16 + g + 8 * r;
      if (t >= live) continue;
      float* dst = a.o32 + ((size_t)(t0 + t) * a.H + h) * a.vdim;
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int c = c0 + wn * (V / 2) + j * 8 + 2 * q;
        if (c < a.vdim) *reinterpret_cast<float2*>(dst + c) = make_float2(acc[j][2 * r] * inv[r], acc[j][2 * r + 1] * inv[r]);
      }
    }
    return;
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float ss = 0.f;  // (columns beyond vdim are zeros)
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      acc[j][2 * r] *= inv[r];
      acc[j][2 * r + 1] *= inv[r];
      ss = fmaf(acc[j][2 * r], acc[j][2 * r], ss);
      ss = fmaf(acc[j][2 * r + 1], acc[j][2 * r + 1], ss);
    }
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    if (q == 0) square[wn][wm * 16 + g + 8 * r] = ss;
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = wm * 16 + g + 8 * r;
    if (t >= live) continue;
    const float norm = 1.f / sqrtf((square[0][t] + square[1][t]) / (float)a.vdim + a.eps);
    const __nv_bfloat16* gate = row0 + (size_t)t * a.ld + 2 * (size_t)a.H * a.dim + (size_t)(a.H + h) * a.vdim;
    __nv_bfloat16* dst = a.out + (size_t)(t0 + t) * a.ldo + (size_t)h * a.vdim;
    const float* gain = a.gain + (size_t)h * a.vdim;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int c = wn * (V / 2) + j * 8 + 2 * q;
      if (c >= a.vdim) continue;
      const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + c));
      const float2 gn = *reinterpret_cast<const float2*>(gain + c);
      *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(acc[j][2 * r] * norm * gn.x * __fdividef(1.f, 1.f + __expf(-z.x)),
                                                        acc[j][2 * r + 1] * norm * gn.y * __fdividef(1.f, 1.f + __expf(-z.y)));
    }
  }
}

// ---- host side -----------------------------------------------------------------------------------------------------

int columns_a_block(int dim) { return dim <= 256 ? 128 : (dim <= 512 ? 64 : 32); }

template <typename T>
int launch_step(const MemoryArgs<T>& a, cudaStream_t stream) {
#define PSB_MM_STEP(PER_, R_, W_)                                                                                              \
  do {                                                                                                                         \
    constexpr int cols = 4 * (32 / R_);                                                                                        \
    const int warps = a.nb > 1 ? W_ : (a.vdim + cols - 1) / cols;                                                              \
    psb_launch(matrix_memory_step_kernel<T, PER_, R_, W_>, dim3(a.nb, a.H, a.items), dim3(warps * 32),                          \
               a.nb > 1 ? 0 : stage_tokens(PER_ * R_) * W_ * cols * sizeof(float), stream, a);                                                 \
  } while (0)
  if (a.dim <= 32) PSB_MM_STEP(4, 8, 8);
  else if (a.dim <= 64) PSB_MM_STEP(8, 8, 8);
  else if (a.dim <= 128) PSB_MM_STEP(16, 8, 8);
  else if (a.dim <= 256) PSB_MM_STEP(16, 16, 16);
  else if (a.dim <= 512) PSB_MM_STEP(32, 16, 8);
  else PSB_MM_STEP(32, 32, 8);
#undef PSB_MM_STEP
  PSB_LAUNCH_CHECK("matrix_memory");
  return 0;
}

template <int D, int V>
int launch_chunks(const MemoryArgs<__nv_bfloat16>& a, float* local_s, float* local_n, float* ends, float* starts, int chunks, cudaStream_t stream) {
  using Z = ChunkShape<D, V>;
  static PsbPerDevice configured;
  if (!configured.get()) {
    if (cudaFuncSetAttribute(matrix_memory_chunk_kernel<D, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, Z::CHUNK_SMEM) != cudaSuccess ||
        cudaFuncSetAttribute(matrix_memory_read_kernel<D, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, Z::READ_SMEM) != cudaSuccess)
      PSB_REFUSE("matrix_memory: cannot raise the shared-memory limit");
    configured.set();
  }
  const dim3 grid((a.vdim + V - 1) / V, a.H, chunks);
  psb_launch(matrix_memory_chunk_kernel<D, V>, grid, dim3(MM_THREADS), (size_t)Z::CHUNK_SMEM, stream, a, local_s, local_n, ends);
  PSB_LAUNCH_CHECK("matrix_memory_chunk");
  const long long threads = (long long)a.H * a.dim * a.vdim / 4 + (long long)a.H * a.dim;
  psb_launch(matrix_memory_starts_kernel, dim3((unsigned)((threads + 255) / 256), a.items), dim3(256), 0, stream, a, local_s, local_n,
             (const float*)ends, starts);
  PSB_LAUNCH_CHECK("matrix_memory_starts");
  psb_launch(matrix_memory_read_kernel<D, V>, grid, dim3(MM_THREADS), (size_t)Z::READ_SMEM, stream, a, (const float*)local_s,
             (const float*)local_n, (const float*)starts);
  PSB_LAUNCH_CHECK("matrix_memory_read");
  return 0;
}

}  // namespace

// (dim, vdim) -> 1 if portions of these sizes can be cut into chunks that run side by side
PSB_API int psb_matrix_memory_chunks_supported(int dim, int vdim) { return dim >= 8 && dim <= 256 && dim % 8 == 0 && vdim >= 8 && vdim % 8 == 0 ? 1 : 0; }

// (proj, dtype, ld, bias_i, bias_f, gain, state, slot_floats, item_start, slots, out, ldo, o32, scratch, items, chunks, H, dim, vdim,
//  nb, num_slots, cap, eps, scale, stream).  nb == 1: ``out`` receives the finished rows; nb > 1: ``o32`` [T, H, vdim] the bare
// read-out.  ``scratch`` (bfloat16 only; or null: token by token): chunks x H x (dim vdim + dim + 3) float32, 16-byte aligned,
// ``chunks`` at least the number of chunks of 64 tokens of the step's portions.
PSB_API int psb_matrix_memory(const void* proj, int dtype, long long ld, const void* bias_i, const void* bias_f, const void* gain,
                              void* state, long long slot_floats, const void* item_start, const void* slots, void* out, long long ldo,
                              void* o32, void* scratch, int items, int chunks, int H, int dim, int vdim, int nb, int num_slots, float cap,
                              float eps, float scale, cudaStream_t stream) {
  if (items < 0 || H < 1 || dim < 1 || dim > 1024 || vdim < 1 || num_slots < 1) PSB_REFUSE("matrix_memory: bad sizes H=%d dim=%d vdim=%d (keys of at most 1024)", H, dim, vdim);
  if (nb != (vdim + columns_a_block(dim) - 1) / columns_a_block(dim)) PSB_REFUSE("matrix_memory: %d copies of the normalizer do not go with sizes %d/%d", nb, dim, vdim);
  if (ld < 2LL * H * (dim + vdim) + 2 * H) PSB_REFUSE("matrix_memory: row stride %lld is shorter than the row", ld);
  if (slot_floats < (long long)H * ((long long)dim * vdim + (long long)nb * dim + nb)) PSB_REFUSE("matrix_memory: a slot of %lld numbers does not hold the state", slot_floats);
  if (!(cap > 0.f) || !(eps > 0.f)) PSB_REFUSE("matrix_memory: cap and eps must be positive");
  if (nb == 1 ? (!out || !gain || ldo < (long long)H * vdim) : !o32) PSB_REFUSE("matrix_memory: no place for the read-out");
  if (H > 65535 || items > 65535 || chunks > 65535) PSB_REFUSE("matrix_memory: too many heads, requests or chunks for one launch");
  if (items == 0) return 0;
  PSB_DISPATCH_DTYPE(dtype, T, {
    MemoryArgs<T> a{};
    a.proj = (const T*)proj; a.ld = ld; a.bias_i = (const float*)bias_i; a.bias_f = (const float*)bias_f; a.gain = (const float*)gain;
    a.state = (float*)state; a.slot_floats = slot_floats; a.item_start = (const int32_t*)item_start; a.slots = (const int32_t*)slots;
    a.out = (T*)out; a.ldo = ldo; a.o32 = (float*)o32; a.items = items; a.H = H; a.dim = dim; a.vdim = vdim; a.nb = nb;
    a.num_slots = num_slots; a.cap = cap; a.eps = eps; a.scale = scale;
    if (!scratch) return launch_step<T>(a, stream);
  });
  if (dtype != PSB_BF16 || !psb_matrix_memory_chunks_supported(dim, vdim) || chunks < items || (((uintptr_t)proj | (uintptr_t)scratch | (uintptr_t)state) & 15) ||
      ld % 8 || ((uintptr_t)out & 3) || ldo % 2 || ((uintptr_t)gain & 7) || slot_floats % 4)
    PSB_REFUSE("matrix_memory: chunks side by side need bfloat16 rows in multiples of eight and aligned operands");
  MemoryArgs<__nv_bfloat16> a{};
  a.proj = (const __nv_bfloat16*)proj; a.ld = ld; a.bias_i = (const float*)bias_i; a.bias_f = (const float*)bias_f; a.gain = (const float*)gain;
  a.state = (float*)state; a.slot_floats = slot_floats; a.item_start = (const int32_t*)item_start; a.slots = (const int32_t*)slots;
  a.out = (__nv_bfloat16*)out; a.ldo = ldo; a.o32 = (float*)o32; a.items = items; a.H = H; a.dim = dim; a.vdim = vdim; a.nb = nb;
  a.num_slots = num_slots; a.cap = cap; a.eps = eps; a.scale = scale;
  const size_t units = (size_t)chunks * H;
  float* local_s = (float*)scratch;
  float* local_n = local_s + units * dim * vdim;
  float* ends = local_n + units * dim;
  float* starts = ends + units * 2;
#define PSB_MM_CHUNKS(D_) (vdim <= 64 ? launch_chunks<D_, 64>(a, local_s, local_n, ends, starts, chunks, stream) \
                                      : launch_chunks<D_, 128>(a, local_s, local_n, ends, starts, chunks, stream))
  if (dim <= 64) return PSB_MM_CHUNKS(64);
  if (dim <= 128) return PSB_MM_CHUNKS(128);
  return PSB_MM_CHUNKS(256);
#undef PSB_MM_CHUNKS
}

// Grouped-query attention over paged keys and values of any head size, for models that list their layers:
// K [page][kv head][16][dk], V [page][kv head][16][dv] (sizes padded to 64), and with pooled blocks their mean keys and
// values [page][kv head][blocks that can end in a page][..], each in the page of its last position.
//
//   kv_append_kernel    folds the projection's slices (or reads bf16 GEMM rows), stores keys and values at their positions
//                       and the queries as rows
//   kv_norm_kernel      the same for heads with biases, norms, rotations, gates and a query temperature, a warp per (row,
//                       head); fills the pooled blocks that end at its rows
//   paged_rows_kernel   split-KV attention of single rows (mma.m16n8k16): a CTA serves up to 16 query heads of one KV head
//                       and one row; its four warps take the pages in turn, each with a cp.async ring and an online
//                       softmax of its own, and meet in shared memory
//   paged_merge_kernel  merge of the splits
//   paged_simple_kernel the same in plain fp32 arithmetic for either element type
//   pool_gather_kernel  pooled keys and values of a batch's prompt segments as contiguous rows
//
// What a score may carry besides (q . k) scale, each optional: a distance bias -slope_h (i - j), or a logarithmic one
// -r1_h ln(1 + r2_h (i - j)); a chunk size, with which a
// position sees the keys of its own chunk only (chunks counted from position 0); a window of positions, and beside it the
// pooled blocks that lie wholly before it; a sink per head, one more term of the
// softmax's denominator that has no key.  Scores, weights and sums are fp32; the weights enter their product as two bf16
// limbs.  What a result may go through: values that were rotated by their positions are turned back by the row's, a gate.
//
// Rotated pairs are neighbours (dimensions 2 i and 2 i + 1): the order of a head's dimensions is the loader's choice.
#include "common.cuh"

using namespace b2;

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }
__device__ __forceinline__ void store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}

// first position a row at `pos` sees
__device__ __forceinline__ int first_key(int pos, int chunk, int window) {
  return chunk > 0 ? pos - pos % chunk : window > 0 ? max(0, pos - window + 1) : 0;
}
// row of the pooled block whose last position is e, in a plane of `slots` blocks per page
__device__ __forceinline__ size_t pool_row(const int* bt, int e, int G, int kh, int slots, int pool) {
  return ((size_t)bt[e >> 4] * G + kh) * slots + (e & 15) / pool;
}

// ------------------------------------------------------------------ keys and values into the pages
struct AppendParams {
  const void* part;        // fp32 [S][M][N], or (rows form) bf16 [M][N]; columns: queries, keys, values
  int S, M, N, nq, G, dk, dv;
  const int *req, *pos, *block_table;
  int max_blocks;
  void *q, *k, *v;         // q [M][nq]
};

// grid (rows, column blocks); a thread owns four columns
template <typename T>
__global__ void __launch_bounds__(256) kv_append_kernel(const AppendParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int m = blockIdx.x, c = (blockIdx.y * 256 + threadIdx.x) * 4;
  if (c >= p.N) return;
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b[8];
  const float* src = reinterpret_cast<const float*>(p.part) + (size_t)m * p.N + c;
#pragma unroll
  for (int s = 0; s < 8; ++s) b[s] = s < p.S ? __ldcg(reinterpret_cast<const float4*>(src + (size_t)s * p.M * p.N)) : a;
#pragma unroll
  for (int s = 0; s < 8; ++s) { a.x += b[s].x; a.y += b[s].y; a.z += b[s].z; a.w += b[s].w; }
  if (c < p.nq) {
    store4(reinterpret_cast<T*>(p.q) + (size_t)m * p.nq + c, a);
    return;
  }
  const int pos = p.pos[m], page = p.block_table[(size_t)p.req[m] * p.max_blocks + (pos >> 4)];
  int j = c - p.nq;
  const int nk = p.G * p.dk, d = j < nk ? p.dk : p.dv;
  T* dst = reinterpret_cast<T*>(j < nk ? p.k : p.v);
  if (j >= nk) j -= nk;
  const int h = j / d;
  store4(dst + (((size_t)page * p.G + h) * 16 + (pos & 15)) * d + (j - h * d), a);
}

// bf16 rows of a GEMM: the queries stay where they are; a thread owns eight columns
__global__ void __launch_bounds__(128) kv_append_rows_kernel(const AppendParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int m = blockIdx.x, nk = p.G * p.dk, n = nk + p.G * p.dv;
  const int pos = p.pos[m], page = p.block_table[(size_t)p.req[m] * p.max_blocks + (pos >> 4)];
  const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.part) + (size_t)m * p.N + p.nq);
  for (int i = threadIdx.x; i < n / 8; i += 128) {
    int j = i * 8;
    const int d = j < nk ? p.dk : p.dv;
    __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(j < nk ? p.k : p.v);
    if (j >= nk) j -= nk;
    const int h = j / d;
    *reinterpret_cast<uint4*>(dst + (((size_t)page * p.G + h) * 16 + (pos & 15)) * d + (j - h * d)) = src[i];
  }
}

// ------------------------------------------------------------------ heads with biases, norms and a query temperature
struct NormParams {
  const float* part;       // [slices][M][N]; columns: queries [H dk] | keys [G dk] | values [G dv] | others
  int slices, M, N, H, G, dk, dv, dim, vdim;
  const float* bias;       // [H dk + G dk + G dv], or null
  const float *q_norm, *k_norm;    // [dk] factors after the division by the root mean square, or null: no such norm
  int v_norm;              // values are divided by their root mean square
  float eps, temp;         // queries times 1 + temp ln(floor((p + 1) / every) + 1)
  int every;
  const int *req, *pos, *block_table;
  int max_blocks;
  void *q, *k, *v;         // q [M][H dk]
  // the rest: the kernel's EXT form
  const float *cos, *sin;  // [positions][rd / 2] rotation of queries and keys behind their norms (rd 0: none)
  const float *vcos, *vsin;        // [positions][vd / 2] rotation of values (vd 0: none)
  int rd, vd;
  int tied;                // values are the keys' columns, without norm and rotation
  int gate_col;            // [H dv] columns whose sigmoid goes to gate [M][H dv] (gate null: none)
  void* gate;
  int pool, slots;         // pool > 0: means of whole blocks of this many positions, `slots` of them per page
  void *pk, *pv;
};

__device__ __forceinline__ float rounded(float v, float) { return v; }
__device__ __forceinline__ float rounded(float v, __nv_bfloat16) { return __bfloat162float(__float2bfloat16(v)); }
__device__ __forceinline__ float4 load4(const float* p) { return __ldcg(reinterpret_cast<const float4*>(p)); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 r = __ldcg(reinterpret_cast<const uint2*>(p));
  return make_float4(bf16_lo(r.x), bf16_hi(r.x), bf16_lo(r.y), bf16_hi(r.y));
}

// NQ: quads of columns per lane; EXT: rotations, tied values, gates, pooled blocks
template <int NQ, typename T, bool EXT>
__global__ void __launch_bounds__(128) kv_norm_kernel(const NormParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int m = blockIdx.x, head = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const bool is_gate = EXT && head >= p.H + 2 * p.G;
  if (head >= p.H + 2 * p.G + (EXT && p.gate ? p.H : 0)) return;
  const bool is_q = head < p.H, is_v = head >= p.H + p.G && !is_gate, same = EXT && is_v && p.tied;
  const int d = is_v || is_gate ? p.dv : p.dk;
  const int col = is_gate ? p.gate_col + (head - p.H - 2 * p.G) * p.dv : same ? (head - p.G) * p.dk
                  : is_v ? (p.H + p.G) * p.dk + (head - p.H - p.G) * p.dv : head * p.dk;
  const long long slice = (long long)p.M * p.N;
  const float* w = is_v || is_gate ? nullptr : is_q ? p.q_norm : p.k_norm;
  // the head's columns of row `row`, normed and rotated
  auto make = [&](int row, int pos, float4 (&x)[NQ]) {
    const float* src = p.part + (size_t)row * p.N + col;
    float ssq = 0.f;
#pragma unroll
    for (int u = 0; u < NQ; ++u) {
      const int c = (u * 32 + lane) * 4;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b[8];
      if (c < d) {
#pragma unroll
        for (int s = 0; s < 8; ++s) b[s] = s < p.slices ? __ldcg(reinterpret_cast<const float4*>(src + s * slice + c)) : a;
#pragma unroll
        for (int s = 0; s < 8; ++s) { a.x += b[s].x; a.y += b[s].y; a.z += b[s].z; a.w += b[s].w; }
        if (p.bias && !is_gate) {
          const float4 w4 = *reinterpret_cast<const float4*>(p.bias + col + c);
          a.x += w4.x; a.y += w4.y; a.z += w4.z; a.w += w4.w;
        }
      }
      x[u] = a;
      ssq += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;      // padding columns are zero
    }
    float r = 1.f;
    if (w || (is_v && p.v_norm)) r = 1.f / sqrtf(warp_sum(ssq) / (float)(is_v ? p.vdim : p.dim) + p.eps);
    if (is_q && p.temp != 0.f) r *= 1.f + p.temp * logf((float)((pos + 1) / p.every) + 1.f);
    const int n2 = !EXT || is_gate || same ? 0 : (is_v ? p.vd : p.rd) / 2;
    const float *cs = (is_v ? p.vcos : p.cos) + (size_t)pos * n2, *sn = (is_v ? p.vsin : p.sin) + (size_t)pos * n2;
#pragma unroll
    for (int u = 0; u < NQ; ++u) {
      const int c = (u * 32 + lane) * 4;
      float4 f = make_float4(r, r, r, r);
      if (w && c < d) {
        const float4 g = *reinterpret_cast<const float4*>(w + c);
        f = make_float4(r * g.x, r * g.y, r * g.z, r * g.w);
      }
      x[u] = make_float4(x[u].x * f.x, x[u].y * f.y, x[u].z * f.z, x[u].w * f.w);
      if (EXT && n2) {
        const int i = c >> 1;
        if (i < n2) {
          const float a = cs[i], b = sn[i];
          x[u] = make_float4(x[u].x * a - x[u].y * b, x[u].y * a + x[u].x * b, x[u].z, x[u].w);
        }
        if (i + 1 < n2) {
          const float a = cs[i + 1], b = sn[i + 1];
          x[u] = make_float4(x[u].x, x[u].y, x[u].z * a - x[u].w * b, x[u].w * a + x[u].z * b);
        }
      }
    }
  };
  const int pos = p.pos[m], h = head - p.H - (is_v ? p.G : 0);
  const int* bt = p.block_table + (size_t)p.req[m] * p.max_blocks;
  float4 x[NQ];
  make(m, pos, x);
  T* dst;
  if (is_q) {
    dst = reinterpret_cast<T*>(p.q) + (size_t)m * p.H * p.dk + col;
  } else if (is_gate) {
    dst = reinterpret_cast<T*>(p.gate) + (size_t)m * p.H * p.dv + col - p.gate_col;
#pragma unroll
    for (int u = 0; u < NQ; ++u)
      x[u] = make_float4(1.f / (1.f + expf(-x[u].x)), 1.f / (1.f + expf(-x[u].y)), 1.f / (1.f + expf(-x[u].z)), 1.f / (1.f + expf(-x[u].w)));
  } else {
    dst = reinterpret_cast<T*>(is_v ? p.v : p.k) + (((size_t)bt[pos >> 4] * p.G + h) * 16 + (pos & 15)) * d;
  }
#pragma unroll
  for (int u = 0; u < NQ; ++u) {
    const int c = (u * 32 + lane) * 4;
    if (c < d) store4(dst + c, x[u]);
  }
  if (!EXT || is_q || is_gate || !p.pool || (pos + 1) % p.pool) return;
  // the block that ends here: the mean of what the cache holds for its positions.  Rows of this step are made again from the
  // projection (another CTA stores them), the others read
  float4 sum[NQ];
#pragma unroll
  for (int u = 0; u < NQ; ++u) sum[u] = make_float4(rounded(x[u].x, T()), rounded(x[u].y, T()), rounded(x[u].z, T()), rounded(x[u].w, T()));
  for (int j = 1; j < p.pool; ++j) {
    const int at = pos - j;
    if (m - j >= 0 && p.req[m - j] == p.req[m] && p.pos[m - j] == at) {
      make(m - j, at, x);
#pragma unroll
      for (int u = 0; u < NQ; ++u) x[u] = make_float4(rounded(x[u].x, T()), rounded(x[u].y, T()), rounded(x[u].z, T()), rounded(x[u].w, T()));
    } else {
      const T* src = reinterpret_cast<const T*>(is_v ? p.v : p.k) + (((size_t)bt[at >> 4] * p.G + h) * 16 + (at & 15)) * d;
#pragma unroll
      for (int u = 0; u < NQ; ++u) {
        const int c = (u * 32 + lane) * 4;
        if (c < d) x[u] = load4(src + c);
      }
    }
#pragma unroll
    for (int u = 0; u < NQ; ++u) { sum[u].x += x[u].x; sum[u].y += x[u].y; sum[u].z += x[u].z; sum[u].w += x[u].w; }
  }
  dst = reinterpret_cast<T*>(is_v ? p.pv : p.pk) + pool_row(bt, pos, p.G, h, p.slots, p.pool) * d;
  const float n = (float)p.pool;
#pragma unroll
  for (int u = 0; u < NQ; ++u) {
    const int c = (u * 32 + lane) * 4;
    if (c < d) store4(dst + c, make_float4(sum[u].x / n, sum[u].y / n, sum[u].z / n, sum[u].w / n));
  }
}

template <int NQ, typename T>
int launch_norm_form(const NormParams& p, dim3 grid, cudaStream_t st) {
  return p.rd || p.vd || p.tied || p.gate || p.pool ? b2_launch(kv_norm_kernel<NQ, T, true>, grid, dim3(128), 0, st, true, p)
                                                    : b2_launch(kv_norm_kernel<NQ, T, false>, grid, dim3(128), 0, st, true, p);
}

template <typename T>
int launch_norm(const NormParams& p, cudaStream_t st) {
  const dim3 grid(p.M, (p.H + 2 * p.G + (p.gate ? p.H : 0) + 3) / 4);
  const int quads = ((p.dk > p.dv ? p.dk : p.dv) + 127) / 128;
  if (quads <= 1) return launch_norm_form<1, T>(p, grid, st);
  if (quads <= 2) return launch_norm_form<2, T>(p, grid, st);
  if (quads <= 4) return launch_norm_form<4, T>(p, grid, st);
  return launch_norm_form<8, T>(p, grid, st);
}

// ------------------------------------------------------------------ pooled rows of prompt segments, one after another
struct GatherParams {
  const int *req, *block;  // [n] slot and block of every row
  const int* block_table;
  int max_blocks, n, G, dk, dv, pool, slots;
  const __nv_bfloat16 *pk, *pv;
  __nv_bfloat16 *k, *v;    // [n][G dk], [n][G dv]
};

__global__ void __launch_bounds__(128) pool_gather_kernel(const GatherParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, e = p.block[r] * p.pool + p.pool - 1, nk = p.G * p.dk, n = nk + p.G * p.dv;
  const int* bt = p.block_table + (size_t)p.req[r] * p.max_blocks;
  for (int i = threadIdx.x * 8; i < n; i += 128 * 8) {
    const bool key = i < nk;
    const int d = key ? p.dk : p.dv, j = key ? i : i - nk, h = j / d;
    const uint4* src = reinterpret_cast<const uint4*>((key ? p.pk : p.pv) + pool_row(bt, e, p.G, h, p.slots, p.pool) * d + (j - h * d));
    *reinterpret_cast<uint4*>(key ? p.k + (size_t)r * nk + j : p.v + (size_t)r * (n - nk) + j) = __ldcg(src);
  }
}

// ------------------------------------------------------------------ what a head's result goes through
struct Finish {
  const float *cos, *sin;  // [positions][half]: pair i is turned back by the row's angle (half 0: none)
  int half;
  const void* gate;        // rows of ldg elements [H][dv], or null
  int ldg;
};

// columns c .. c + 3 of head h (`col`: of the row)
template <typename T>
__device__ __forceinline__ float4 finish(const Finish& f, float4 v, int m, int pos, int c, int col) {
  const int i = c >> 1;
  if (i < f.half) {
    const float a = f.cos[(size_t)pos * f.half + i], b = f.sin[(size_t)pos * f.half + i];
    v = make_float4(v.x * a + v.y * b, v.y * a - v.x * b, v.z, v.w);
  }
  if (i + 1 < f.half) {
    const float a = f.cos[(size_t)pos * f.half + i + 1], b = f.sin[(size_t)pos * f.half + i + 1];
    v = make_float4(v.x, v.y, v.z * a + v.w * b, v.w * a - v.z * b);
  }
  if (f.gate) {
    const float4 g = load4(reinterpret_cast<const T*>(f.gate) + (size_t)m * f.ldg + col);
    v = make_float4(v.x * g.x, v.y * g.y, v.z * g.z, v.w * g.w);
  }
  return v;
}

// ------------------------------------------------------------------ attention of single rows (tensor cores)
struct RowsParams {
  const __nv_bfloat16 *q, *k, *v;    // q: rows of ldq elements, the first H dk of each
  const int *req, *pos, *block_table;
  int ldq, max_blocks, H, G, nsplit, chunk;
  float scale_log2;
  const float *slope2, *sink2;       // [H] times log2 e, or null
  const float *r1, *r2;              // [H] logarithmic distance bias (in powers of two: r1 log2(1 + r2 distance)), or null
  float *o_part, *ml_part;           // [M][H][nsplit][dv], [M][H][nsplit][2]
  __nv_bfloat16* out;                // rows of ldo elements [H][dv], written when nsplit is 1
  int ldo;
  float mult;                        // factor of the result
  int window, pool, slots;           // pool > 0: pooled blocks before the window
  const __nv_bfloat16 *pk, *pv;
  Finish fin;
};

constexpr int kWarps = 4;

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}

// NDK / NDV: blocks of 64 dims of a key / value.  A page of one head is kept as blocks of 16 keys x 128 bytes whose
// 16-byte pieces sit at (piece XOR key mod 8).
template <int NDK, int NDV>
struct RowsForm {
  static constexpr int PAGE = (NDK + NDV) * 2048;
  static constexpr int STAGES = NDK + NDV <= 4 ? 3 : 2;
  static constexpr int RING = kWarps * STAGES * PAGE;
  static constexpr int MERGE = kWarps * 16 * (NDV * 64 + 4) * 4;
  static constexpr int SMEM = RING > MERGE ? RING : MERGE;
};

// POOL: the keys are the pooled blocks before the window, in tiles of 16, and then the window's pages
template <int NDK, int NDV, bool POOL>
__global__ void __launch_bounds__(kWarps * 32) paged_rows_kernel(const RowsParams p) {
  using F = RowsForm<NDK, NDV>;
  constexpr int dk = NDK * 64, dv = NDV * 64, ST = F::STAGES;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ float s_m[kWarps][16], s_l[kWarps][16];
  const int m = blockIdx.x, split = blockIdx.y, R = p.H / p.G, tiles = (R + 15) / 16;
  const int kh = blockIdx.z / tiles, r0 = (blockIdx.z % tiles) * 16, nr = min(16, R - r0), h0 = kh * R + r0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  pdl_launch_dependents();
  pdl_wait();
  const int pos = p.pos[m], lo = first_key(pos, p.chunk, p.window);
  const int* bt = p.block_table + (size_t)p.req[m] * p.max_blocks;
  const int n_pool = POOL ? lo / p.pool : 0, tiles_pool = (n_pool + 15) >> 4;
  const int page_lo = (lo >> 4) - tiles_pool, pages = (pos >> 4) + 1 - page_lo, pps = (pages + p.nsplit - 1) / p.nsplit;
  const int pg0 = split * pps, pg1 = min(pages, pg0 + pps);
  const int n = pg1 > pg0 + warp ? (pg1 - pg0 - warp + kWarps - 1) / kWarps : 0;      // this warp's pages: pg0 + warp + 4 i
  const uint32_t ring = smem_u32(smem) + warp * ST * F::PAGE;
  auto issue = [&](int i) {
    const int tile = pg0 + warp + kWarps * i;
    if (POOL && i < n && tile < tiles_pool) {
      const uint32_t dst = ring + (i % ST) * F::PAGE;
      // past the last block: that one again
      const unsigned long long at = pool_row(bt, min(tile * 16 + (lane & 15), n_pool - 1) * p.pool + p.pool - 1, p.G, kh, p.slots, p.pool);
#pragma unroll
      for (int u = 0; u < 4 * NDK; ++u) {
        const int j = u * 32 + lane, row = j / (NDK * 8), pc = j % (NDK * 8);
        cp16(dst + (pc >> 3) * 2048 + row * 128 + (((pc & 7) ^ (row & 7)) << 4), p.pk + __shfl_sync(0xffffffffu, at, row) * dk + pc * 8);
      }
#pragma unroll
      for (int u = 0; u < 4 * NDV; ++u) {
        const int j = u * 32 + lane, row = j / (NDV * 8), pc = j % (NDV * 8);
        cp16(dst + (NDK + (pc >> 3)) * 2048 + row * 128 + (((pc & 7) ^ (row & 7)) << 4), p.pv + __shfl_sync(0xffffffffu, at, row) * dv + pc * 8);
      }
    } else if (i < n) {
      const int page = bt[page_lo + tile];
      const uint32_t dst = ring + (i % ST) * F::PAGE;
      const __nv_bfloat16* ks = p.k + ((size_t)page * p.G + kh) * 16 * dk;
      const __nv_bfloat16* vs = p.v + ((size_t)page * p.G + kh) * 16 * dv;
#pragma unroll
      for (int u = 0; u < 4 * NDK; ++u) {
        const int j = u * 32 + lane, row = j / (NDK * 8), pc = j % (NDK * 8);
        cp16(dst + (pc >> 3) * 2048 + row * 128 + (((pc & 7) ^ (row & 7)) << 4), ks + j * 8);
      }
#pragma unroll
      for (int u = 0; u < 4 * NDV; ++u) {
        const int j = u * 32 + lane, row = j / (NDV * 8), pc = j % (NDV * 8);
        cp16(dst + (NDK + (pc >> 3)) * 2048 + row * 128 + (((pc & 7) ^ (row & 7)) << 4), vs + j * 8);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < ST; ++i) issue(i);
  // the queries' fragments; rows past the group's heads are zero
  uint32_t qa[NDK * 4][4];
#pragma unroll
  for (int k = 0; k < NDK * 4; ++k)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = g + 8 * (e & 1), c = k * 16 + 2 * t + 8 * (e >> 1);
      qa[k][e] = r < nr ? *reinterpret_cast<const uint32_t*>(p.q + (size_t)m * p.ldq + (h0 + r) * dk + c) : 0u;
    }
  float slope[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};      // slope: r1 of a logarithmic bias
  if (p.slope2 || p.r1) {
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int hd = h0 + min(g + 8 * hf, nr - 1);
      slope[hf] = p.r1 ? p.r1[hd] : p.slope2[hd];
      if (p.r1) r2[hf] = p.r2[hd];
    }
  }
  float o[NDV * 8][4];
#pragma unroll
  for (int j = 0; j < NDV * 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const uint32_t sw = lane & 7, mi = lane >> 3;
  for (int i = 0; i < n; ++i) {
    asm volatile("cp.async.wait_group %0;" ::"n"(ST - 1) : "memory");
    __syncwarp();
    const uint32_t kb = ring + (i % ST) * F::PAGE, vb = kb + NDK * 2048;
    float s[2][2][4];          // two chains per key half
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int j = 0; j < 2; ++j) s[a][j][0] = s[a][j][1] = s[a][j][2] = s[a][j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < NDK * 2; ++kk)        // 32 dims
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        uint32_t b[4];
        ldsm_x4(kb + (kk >> 1) * 2048 + (8 * j + (lane & 7)) * 128 + (((4 * (kk & 1) + mi) ^ sw) << 4), b);
        mma_bf16_16816(s[0][j], qa[2 * kk][0], qa[2 * kk][1], qa[2 * kk][2], qa[2 * kk][3], b[0], b[1]);
        mma_bf16_16816(s[1][j], qa[2 * kk + 1][0], qa[2 * kk + 1][1], qa[2 * kk + 1][2], qa[2 * kk + 1][3], b[2], b[3]);
      }
    const int tile = pg0 + warp + kWarps * i;
    const bool pooled = POOL && tile < tiles_pool;
    const int key0 = pooled ? tile * 16 : (page_lo + tile) * 16, first = pooled ? 0 : lo, last = pooled ? n_pool - 1 : pos;
    float x[2][4], top[2] = {mx[0], mx[1]};
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = key0 + 8 * j + 2 * t + (e & 1);
        float away = (float)(key - pos);
        if (p.r1) away = -__log2f(fmaf(-r2[e >> 1], fminf(away, 0.f), 1.f));
        const float v = fmaf(slope[e >> 1], away, (s[0][j][e] + s[1][j][e]) * p.scale_log2);
        x[j][e] = key >= first && key <= last ? v : -INFINITY;
        top[e >> 1] = fmaxf(top[e >> 1], x[j][e]);
      }
    float corr[2];
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      top[hf] = fmaxf(top[hf], __shfl_xor_sync(0xffffffffu, top[hf], 1));
      top[hf] = fmaxf(top[hf], __shfl_xor_sync(0xffffffffu, top[hf], 2));
      corr[hf] = exp2f(mx[hf] - top[hf]);        // every page of the loop has a visible key: top is finite
      l[hf] *= corr[hf];
      mx[hf] = top[hf];
    }
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const float e0 = exp2f(x[j][2 * hf] - mx[hf]), e1 = exp2f(x[j][2 * hf + 1] - mx[hf]);
        l[hf] += e0 + e1;
        const uint32_t hi = pack_bf16(e0, e1);
        ph[2 * j + hf] = hi;
        pl[2 * j + hf] = pack_bf16(e0 - bf16_lo(hi), e1 - bf16_hi(hi));
      }
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int j = 0; j < NDV * 8; ++j) {
        o[j][0] *= corr[0]; o[j][1] *= corr[0]; o[j][2] *= corr[1]; o[j][3] *= corr[1];
      }
    }
#pragma unroll
    for (int j = 0; j < NDV * 8; j += 2) {       // 16 dims: keys 0-7 / 8-15 of dims 8 j, then of dims 8 (j + 1)
      uint32_t b[4];
      ldsm_x4_trans(vb + (j >> 3) * 2048 + (8 * (mi & 1) + (lane & 7)) * 128 + ((((j & 7) + (mi >> 1)) ^ sw) << 4), b);
      mma_bf16_16816(o[j], ph[0], ph[1], ph[2], ph[3], b[0], b[1]);
      mma_bf16_16816(o[j + 1], ph[0], ph[1], ph[2], ph[3], b[2], b[3]);
      mma_bf16_16816(o[j], pl[0], pl[1], pl[2], pl[3], b[0], b[1]);
      mma_bf16_16816(o[j + 1], pl[0], pl[1], pl[2], pl[3], b[2], b[3]);
    }
    __syncwarp();
    issue(i + ST);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    l[hf] += __shfl_xor_sync(0xffffffffu, l[hf], 1);
    l[hf] += __shfl_xor_sync(0xffffffffu, l[hf], 2);
    if (t == 0) {
      s_m[warp][g + 8 * hf] = mx[hf];
      s_l[warp][g + 8 * hf] = l[hf];
    }
  }
  __syncthreads();             // the rings are free: the warps' accumulators take their place
  float* acc = reinterpret_cast<float*>(smem);           // [warp][16][dv + 4]
#pragma unroll
  for (int j = 0; j < NDV * 8; ++j)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf)
      *reinterpret_cast<float2*>(acc + (warp * 16 + g + 8 * hf) * (dv + 4) + 8 * j + 2 * t) = make_float2(o[j][2 * hf], o[j][2 * hf + 1]);
  __syncthreads();
  for (int i = threadIdx.x; i < nr * (dv / 4); i += kWarps * 32) {
    const int r = i / (dv / 4), c = (i - r * (dv / 4)) * 4;
    float top = -INFINITY, sum = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) top = fmaxf(top, s_m[w][r]);
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float e = s_m[w][r] == -INFINITY ? 0.f : exp2f(s_m[w][r] - top);
      const float4 v = *reinterpret_cast<const float4*>(acc + (w * 16 + r) * (dv + 4) + c);
      sum += e * s_l[w][r];
      a.x = fmaf(e, v.x, a.x); a.y = fmaf(e, v.y, a.y); a.z = fmaf(e, v.z, a.z); a.w = fmaf(e, v.w, a.w);
    }
    if (p.nsplit == 1) {
      const float inv = p.mult / (sum + (p.sink2 ? exp2f(p.sink2[h0 + r] - top) : 0.f));
      store4(p.out + (size_t)m * p.ldo + (h0 + r) * dv + c,
             finish<__nv_bfloat16>(p.fin, make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv), m, pos, c, (h0 + r) * dv + c));
    } else {
      const size_t row = ((size_t)m * p.H + h0 + r) * p.nsplit + split;
      *reinterpret_cast<float4*>(p.o_part + row * dv + c) = a;
      if (c == 0) {
        p.ml_part[2 * row] = top;
        p.ml_part[2 * row + 1] = sum;
      }
    }
  }
}

// ------------------------------------------------------------------ merge of the splits: one CTA per (row, head)
struct MergeParams {
  const float *o_part, *ml_part;
  int H, nsplit, dv;
  const float* sink2;
  __nv_bfloat16* out;
  int ldo;
  float mult;
  const int* pos;
  Finish fin;
};

__global__ void __launch_bounds__(128) paged_merge_kernel(const MergeParams p) {
  __shared__ float wt[64];
  __shared__ __align__(16) float4 red[128];
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = blockIdx.x;
  const int h = blockIdx.x % p.H, tid = threadIdx.x, quads = p.dv / 4, groups = 128 / quads;
  if (tid < 32) {               // nsplit <= 64: two splits per lane
    float mx[2], l[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = tid + 32 * i;
      const float2 v = s < p.nsplit ? __ldcg(reinterpret_cast<const float2*>(p.ml_part) + row * p.nsplit + s) : make_float2(-INFINITY, 0.f);
      mx[i] = v.x;
      l[i] = v.y;
    }
    const float top = warp_max(fmaxf(mx[0], mx[1]));
    float e[2], sum = 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      e[i] = mx[i] == -INFINITY ? 0.f : exp2f(mx[i] - top);
      sum += e[i] * l[i];
    }
    const float inv = p.mult / (warp_sum(sum) + (p.sink2 ? exp2f(p.sink2[h] - top) : 0.f));
    wt[tid] = e[0] * inv;
    wt[tid + 32] = e[1] * inv;
  }
  const int grp = tid / quads, c = (tid % quads) * 4;
  const float* o = p.o_part + row * p.nsplit * p.dv + c;
  float4 v[8], a = make_float4(0.f, 0.f, 0.f, 0.f);
  auto fetch = [&](int s0) {
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      const int s = s0 + u * groups;
      v[u] = grp < groups && s < p.nsplit ? __ldcg(reinterpret_cast<const float4*>(o + (size_t)s * p.dv)) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  fetch(grp);
  __syncthreads();
  for (int s0 = grp; s0 < p.nsplit; s0 += 8 * groups) {
    if (s0 != grp) fetch(s0);
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      const int s = s0 + u * groups;
      const float w = s < p.nsplit ? wt[s] : 0.f;
      a.x = fmaf(w, v[u].x, a.x); a.y = fmaf(w, v[u].y, a.y); a.z = fmaf(w, v[u].z, a.z); a.w = fmaf(w, v[u].w, a.w);
    }
  }
  red[tid] = a;
  __syncthreads();
  if (tid < quads) {
    for (int i = 1; i < groups; ++i) {
      const float4 b = red[tid + i * quads];
      a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w;
    }
    const int m = (int)(row / p.H);
    store4(p.out + (size_t)m * p.ldo + h * p.dv + c, finish<__nv_bfloat16>(p.fin, a, m, p.pos[m], c, h * p.dv + c));
  }
}

// ------------------------------------------------------------------ the same in plain fp32 arithmetic
struct SimpleParams {
  const void *q, *k, *v;
  const int *req, *pos, *block_table;
  int ldq, max_blocks, H, G, dk, dv, chunk;
  float scale;
  const float *slope2, *sink2, *r1, *r2;
  void* out;                   // rows of ldo elements [H][dv]
  int ldo;
  float mult;
  int window, pool, slots;
  const void *pk, *pv;
  Finish fin;
};
constexpr int kSimpleDims = 16;    // value dims per thread: dv <= 2048
constexpr float kLn2 = 0.6931471805599453f;

template <typename T>
__global__ void __launch_bounds__(128) paged_simple_kernel(const SimpleParams p) {
  extern __shared__ float qs[];      // [dk]
  __shared__ float sc[128];
  __shared__ const T *k_of[128], *v_of[128];
  pdl_launch_dependents();
  pdl_wait();
  const int m = blockIdx.x, h = blockIdx.y, kh = h / (p.H / p.G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos = p.pos[m];
  const int* bt = p.block_table + (size_t)p.req[m] * p.max_blocks;
  const float slope = p.slope2 ? p.slope2[h] * kLn2 : 0.f, r1 = p.r1 ? p.r1[h] : 0.f, r2 = p.r1 ? p.r2[h] : 0.f;
  for (int i = tid; i < p.dk; i += 128) qs[i] = to_f(reinterpret_cast<const T*>(p.q)[(size_t)m * p.ldq + h * p.dk + i]);
  float o[kSimpleDims];
#pragma unroll
  for (int i = 0; i < kSimpleDims; ++i) o[i] = 0.f;
  float mx = -INFINITY, l = 0.f;
  // keys: the pooled blocks before the window (places below `lo`, counted down to lo - n_pool), then positions
  const int lo = first_key(pos, p.chunk, p.window), n_pool = p.pool ? lo / p.pool : 0;
  for (int k0 = lo - n_pool; k0 <= pos; k0 += 128) {
    const int n = min(128, pos + 1 - k0);
    __syncthreads();
    if (tid < n) {
      const int key = k0 + tid;
      if (key < lo) {
        const size_t r = pool_row(bt, (key - lo + n_pool) * p.pool + p.pool - 1, p.G, kh, p.slots, p.pool);
        k_of[tid] = reinterpret_cast<const T*>(p.pk) + r * p.dk;
        v_of[tid] = reinterpret_cast<const T*>(p.pv) + r * p.dv;
      } else {
        const size_t r = ((size_t)bt[key >> 4] * p.G + kh) * 16 + (key & 15);
        k_of[tid] = reinterpret_cast<const T*>(p.k) + r * p.dk;
        v_of[tid] = reinterpret_cast<const T*>(p.v) + r * p.dv;
      }
    }
    __syncthreads();
    for (int j = warp; j < n; j += 4) {
      const T* c = k_of[j];
      float s = 0.f;
      for (int d = lane; d < p.dk; d += 32) s = fmaf(qs[d], to_f(c[d]), s);
      s = warp_sum(s);
      const float away = (float)(pos - k0 - j);
      if (lane == 0) sc[j] = s * p.scale - (p.r1 ? r1 * log1pf(r2 * away) : slope * away);
    }
    __syncthreads();
    float mn = mx;
    for (int j = 0; j < n; ++j) mn = fmaxf(mn, sc[j]);
    const float corr = expf(mx - mn);
    mx = mn;
    l *= corr;
#pragma unroll
    for (int i = 0; i < kSimpleDims; ++i) o[i] *= corr;
    for (int j = 0; j < n; ++j) {
      const float w = expf(sc[j] - mx);
      l += w;
      const T* c = v_of[j];
#pragma unroll
      for (int i = 0; i < kSimpleDims; ++i)
        if (tid + 128 * i < p.dv) o[i] = fmaf(w, to_f(c[tid + 128 * i]), o[i]);
    }
  }
  if (p.sink2) l += expf(p.sink2[h] * kLn2 - mx);
#pragma unroll
  for (int i = 0; i < kSimpleDims; ++i) {
    const int d = tid + 128 * i;
    float y = o[i] / l * p.mult;
    if (p.fin.half) {
      const float other = __shfl_xor_sync(0xffffffffu, y, 1);        // the pair's other dimension
      if ((d >> 1) < p.fin.half) {
        const float a = p.fin.cos[(size_t)pos * p.fin.half + (d >> 1)], b = p.fin.sin[(size_t)pos * p.fin.half + (d >> 1)];
        y = d & 1 ? y * a - other * b : y * a + other * b;
      }
    }
    if (d >= p.dv) continue;
    if (p.fin.gate) y *= to_f(reinterpret_cast<const T*>(p.fin.gate)[(size_t)m * p.fin.ldg + h * p.dv + d]);
    reinterpret_cast<T*>(p.out)[(size_t)m * p.ldo + h * p.dv + d] = from_f<T>(y);
  }
}

template <int NDK, int NDV, bool POOL>
int launch_rows_form(const RowsParams& p, int M, cudaStream_t st) {
  using F = RowsForm<NDK, NDV>;
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(paged_rows_kernel<NDK, NDV, POOL>, cudaFuncAttributeMaxDynamicSharedMemorySize, F::SMEM);
    if (e != cudaSuccess) return (int)e;
    configured[dev & 63] = true;
  }
  return b2_launch(paged_rows_kernel<NDK, NDV, POOL>, dim3(M, p.nsplit, p.G * ((p.H / p.G + 15) / 16)), dim3(kWarps * 32), F::SMEM,
                   st, true, p);
}

template <int NDK, int NDV>
int launch_rows(const RowsParams& p, int M, cudaStream_t st) {
  return p.pool ? launch_rows_form<NDK, NDV, true>(p, M, st) : launch_rows_form<NDK, NDV, false>(p, M, st);
}

template <int NDK>
int launch_rows_dv(const RowsParams& p, int M, int ndv, cudaStream_t st) {
  switch (ndv) {
    case 1: return launch_rows<NDK, 1>(p, M, st);
    case 2: return launch_rows<NDK, 2>(p, M, st);
    case 3: return launch_rows<NDK, 3>(p, M, st);
    case 4: return launch_rows<NDK, 4>(p, M, st);
  }
  return -1;
}

}  // namespace

// part: fp32 [S][M][N] (rows_form 0), or bf16 [M][N] (rows_form 1: q unused).  N = nq + G (dk + dv), or nq alone.
extern "C" int b2_kv_append(const void* part, int rows_form, int S, int M, int nq, int G, int dk, int dv, int with_kv,
                            const int* req, const int* pos, const int* block_table, int max_blocks, void* q, void* k, void* v,
                            int f32, void* stream) {
  if (M < 1 || S < 1 || S > 8 || nq % 64 || dk % 64 || dv % 64) return -1;
  AppendParams p{part, S, M, nq + (with_kv ? G * (dk + dv) : 0), nq, G, dk, dv, req, pos, block_table, max_blocks, q, k, v};
  cudaStream_t st = (cudaStream_t)stream;
  if (rows_form) return b2_launch(kv_append_rows_kernel, dim3(M), dim3(128), 0, st, true, p);
  const dim3 grid(M, (p.N / 4 + 255) / 256);
  return f32 ? b2_launch(kv_append_kernel<float>, grid, dim3(256), 0, st, true, p)
             : b2_launch(kv_append_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, true, p);
}

// What a call's keys and results are beyond [page][kv head][16]: see NormParams, RowsParams and Finish.  Host structure, passed
// by address; null: none of it.
struct B2AttnExtra {
  const float *cos, *sin, *vcos, *vsin;
  int rd, vd, tied, gate_col;
  void* gate;
  int ldg, window, pool, slots;
  void *pk, *pv;
};

static bool extra_ok(const B2AttnExtra& x, int dk, int dv) {
  if (x.rd < 0 || x.rd % 2 || x.rd > dk || x.vd < 0 || x.vd % 2 || x.vd > dv || x.window < 0 || x.pool < 0) return false;
  if ((x.rd && (!x.cos || !x.sin)) || (x.vd && (!x.vcos || !x.vsin)) || (x.tied && dk != dv)) return false;
  return !x.pool || (x.window > 0 && x.pk && x.pv && x.slots >= (15 + x.pool) / x.pool);
}

// Heads with biases, norms, rotations and a query temperature (see NormParams): fp32 slices [slices][M][N], whose first columns
// are q | k | v (tied: q | k), to query rows and pages.
extern "C" int b2_kv_norm(const float* part, int slices, int M, int N, int H, int G, int dk, int dv, int dim, int vdim, const float* bias,
                          const float* q_norm, const float* k_norm, int v_norm, float eps, float temp, int every, const int* req,
                          const int* pos, const int* block_table, int max_blocks, void* q, void* k, void* v, int f32,
                          const B2AttnExtra* extra, void* stream) {
  const B2AttnExtra x = extra ? *extra : B2AttnExtra{};
  const int own = H * dk + G * (x.tied ? dk : dk + dv);
  if (M < 1 || slices < 1 || slices > 8 || H < 1 || G < 1 || dk % 64 || dv % 64 || dk > 1024 || dv > 1024 || N % 4 ||
      N < own || every < 1 || dim < 1 || vdim < 1 || !extra_ok(x, dk, dv) || (x.gate && (x.gate_col < own || x.gate_col % 4 || x.gate_col + H * dv > N)))
    return -1;
  NormParams p{part, slices, M, N, H, G, dk, dv, dim, vdim, bias, q_norm, k_norm, v_norm, eps, temp, every, req, pos, block_table,
               max_blocks, q, k, v, x.cos, x.sin, x.vcos, x.vsin, x.rd, x.vd, x.tied, x.gate_col, x.gate, x.pool, x.slots, x.pk, x.pv};
  return f32 ? launch_norm<float>(p, (cudaStream_t)stream) : launch_norm<__nv_bfloat16>(p, (cudaStream_t)stream);
}

// Rows (req[i], block[i]) of the pooled planes to k [n][G dk] and v [n][G dv].
extern "C" int b2_pool_gather(const int* req, const int* block, int n, const int* block_table, int max_blocks, int G, int dk, int dv,
                              int pool, int slots, const void* pk, const void* pv, void* k, void* v, void* stream) {
  if (n < 1 || dk % 8 || dv % 8 || pool < 1 || slots < (15 + pool) / pool) return -1;
  GatherParams p{req, block, block_table, max_blocks, n, G, dk, dv, pool, slots, (const __nv_bfloat16*)pk, (const __nv_bfloat16*)pv,
                 (__nv_bfloat16*)k, (__nv_bfloat16*)v};
  return b2_launch(pool_gather_kernel, dim3(n), dim3(128), 0, (cudaStream_t)stream, true, p);
}

// 1 when the tensor-core row kernel covers the head sizes
extern "C" int b2_paged_rows_ok(int dk, int dv) { return dk % 64 == 0 && dv % 64 == 0 && dk >= 64 && dv >= 64 && dk <= 256 && dv <= 256; }

extern "C" int b2_paged_rows(const void* q, int ldq, const void* k, const void* v, int M, int H, int G, int dk, int dv, const int* req,
                             const int* pos, const int* block_table, int max_blocks, int nsplit, int chunk, float scale,
                             const float* slope2, const float* sink2, const float* r1, const float* r2, float* o_part, float* ml_part,
                             void* out, int ldo, float mult, const B2AttnExtra* extra, void* stream) {
  const B2AttnExtra x = extra ? *extra : B2AttnExtra{};
  if (M < 1 || H % G || nsplit < 1 || nsplit > 64 || !b2_paged_rows_ok(dk, dv) || chunk < 0 || ldq < H * dk || ldq % 2 || ldo < H * dv ||
      ldo % 4 || (r1 && !r2) || !extra_ok(x, dk, dv) || (x.window && chunk) || (x.pool && (slope2 || r1)) || (x.gate && (x.ldg < H * dv || x.ldg % 4)))
    return -1;
  const Finish fin{x.vcos, x.vsin, x.vd / 2, x.gate, x.ldg};
  RowsParams p{(const __nv_bfloat16*)q, (const __nv_bfloat16*)k, (const __nv_bfloat16*)v, req, pos, block_table, ldq, max_blocks, H, G,
               nsplit, chunk, scale * 1.4426950408889634f, slope2, sink2, r1, r2, o_part, ml_part, (__nv_bfloat16*)out, ldo, mult,
               x.window, x.pool, x.slots, (const __nv_bfloat16*)x.pk, (const __nv_bfloat16*)x.pv, fin};
  cudaStream_t st = (cudaStream_t)stream;
  int rc = -1;
  switch (dk / 64) {
    case 1: rc = launch_rows_dv<1>(p, M, dv / 64, st); break;
    case 2: rc = launch_rows_dv<2>(p, M, dv / 64, st); break;
    case 3: rc = launch_rows_dv<3>(p, M, dv / 64, st); break;
    case 4: rc = launch_rows_dv<4>(p, M, dv / 64, st); break;
  }
  if (rc || nsplit == 1) return rc;
  MergeParams mp{o_part, ml_part, H, nsplit, dv, sink2, (__nv_bfloat16*)out, ldo, mult, pos, fin};
  return b2_launch(paged_merge_kernel, dim3(M * H), dim3(128), 0, st, true, mp);
}

extern "C" int b2_paged_simple(const void* q, int ldq, const void* k, const void* v, int M, int H, int G, int dk, int dv, const int* req,
                               const int* pos, const int* block_table, int max_blocks, int chunk, float scale,
                               const float* slope2, const float* sink2, const float* r1, const float* r2, void* out, int ldo, float mult,
                               int f32, const B2AttnExtra* extra, void* stream) {
  const B2AttnExtra x = extra ? *extra : B2AttnExtra{};
  if (M < 1 || H % G || H > 65535 || dv > 128 * kSimpleDims || dk > 8192 || chunk < 0 || ldo < H * dv || (r1 && !r2) || !extra_ok(x, dk, dv) ||
      (x.window && chunk) || (x.pool && (slope2 || r1)) || (x.gate && x.ldg < H * dv))
    return -1;
  SimpleParams p{q, k, v, req, pos, block_table, ldq, max_blocks, H, G, dk, dv, chunk, scale, slope2, sink2, r1, r2, out, ldo, mult,
                 x.window, x.pool, x.slots, x.pk, x.pv, {x.vcos, x.vsin, x.vd / 2, x.gate, x.ldg}};
  const size_t smem = (size_t)dk * 4;
  return f32 ? b2_launch(paged_simple_kernel<float>, dim3(M, H), dim3(128), smem, (cudaStream_t)stream, true, p)
             : b2_launch(paged_simple_kernel<__nv_bfloat16>, dim3(M, H), dim3(128), smem, (cudaStream_t)stream, true, p);
}

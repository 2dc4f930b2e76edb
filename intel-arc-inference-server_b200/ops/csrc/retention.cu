// Matrix-memory recurrence with a fixed decay per head (retention): per head a state S [dk][dv], fp32, one per slot.
//
//   S <- decay S + k v^T,   o = S^T q;   out = o / rms(o) * silu(z_g)         rms over the head's value dims
//
// Queries and keys are rotated by their positions (pairs of neighbouring dimensions), keys scaled by dim^-1/2.
//
//   retention_step_kernel   rows in order, one token at a time: a cluster of dv / 64 CTAs per (sequence, head) folds the
//                           projection's slices, rotates, updates the state and writes the gated output; either element type
//   retention_kv_kernel     prompt segments, every chunk of 128 rows by itself: sum_j decay^(last - j) k_j v_j^T
//   retention_scan_kernel   prompt segments: the state ahead of every chunk, element by element
//   retention_chunk_kernel  prompt segments, every chunk by itself: decay^(i + 1) S^T q_i + sum_{j <= i} decay^(i - j) (k_j . q_i) v_j
//   retention_out_kernel    head norm and gate where a head's value dims are spread over several CTAs
//
// Only the scan walks a segment, and it moves the states alone: the products of all chunks run side by side.  Rotated queries
// and keys, the state and the decayed products enter their products as two bf16 limbs, values as the projection's bf16.
//
// A sequence's first row (position 0) starts from a zero state whatever its slot holds.
#include "common.cuh"

#include <cooperative_groups.h>

using namespace b2;
namespace cg = cooperative_groups;

namespace {

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

struct RetentionParams {
  const float* part;      // [slices][M][N]; columns from col: q [H dk] | k [H dk] | v [H dv] | g [H dv]
  int slices, M, N, col, H, dk, dv, vdim;
  const int *req, *pos;
  const float *cos, *sin; // [positions][half]
  int half;
  float k_scale, eps, mult;
  const float* decay;     // [2][H]: decay, log2 of it
  float* state;           // [slots][H][dk][dv]
  void* out;              // rows of ldo elements, [H dv] of them written, times mult
  int ldo;
  // prompt segments
  const int* segs;        // [n][4]: first row, rows, slot, first chunk (counted over all segments)
  float* kv;              // [chunks][H][dk][dv]
  float* raw;             // [M][H dv], or null: a CTA has all value dims of a head
};

// dims c .. c + 3 of a row at `pos`
__device__ __forceinline__ float4 rotated(const RetentionParams& p, float4 x, int pos, int c) {
  const int i = c >> 1;
  const float *cs = p.cos + (size_t)pos * p.half + i, *sn = p.sin + (size_t)pos * p.half + i;
  if (i < p.half) x = make_float4(x.x * cs[0] - x.y * sn[0], x.y * cs[0] + x.x * sn[0], x.z, x.w);
  if (i + 1 < p.half) x = make_float4(x.x, x.y, x.z * cs[1] - x.w * sn[1], x.w * cs[1] + x.z * sn[1]);
  return x;
}

// ------------------------------------------------------------------ one token at a time
// KB: blocks of 64 key dims.  256 threads: 16 groups of 4 value columns x 16 groups of key dims (d = 16 i + group)
template <int KB, typename T>
__global__ void __launch_bounds__(256) retention_step_kernel(const RetentionParams p) {
  constexpr int dk = KB * 64, NS = KB * 4;
  __shared__ __align__(16) float s_q[dk], s_k[dk], s_v[64], s_g[64], s_red[16][64], s_sum[2];
  __shared__ float s_ssq;
  const int vb = blockIdx.x, nvb = gridDim.x, h = blockIdx.y, row0 = blockIdx.z;
  const int tid = threadIdx.x, grp = tid >> 4, c = (tid & 15) * 4;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.req[row0];
  if (row0 > 0 && p.req[row0 - 1] == slot) return;        // the whole cluster leaves: another CTA walks this sequence
  float* st = p.state + ((size_t)slot * p.H + h) * dk * p.dv + vb * 64 + c;
  float4 S[NS];
  const bool fresh = p.pos[row0] == 0;
#pragma unroll
  for (int i = 0; i < NS; ++i)
    S[i] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : __ldcg(reinterpret_cast<const float4*>(st + (size_t)(16 * i + grp) * p.dv));
  const int Hk = p.H * dk, Hv = p.H * p.dv;
  const float keep = p.decay[h];
  cg::cluster_group cl = cg::this_cluster();
  for (int row = row0; row < p.M && p.req[row] == slot; ++row) {
    __syncthreads();            // the row before is done with the shared rows
    const int pos = p.pos[row];
    // q, k, v, g of this head and block: one quad per thread, slices folded
    constexpr int quads = (2 * dk + 128) / 4;
    for (int u = tid; u < quads; u += 256) {
      const int e = u * 4;
      int col;
      float* dst;
      if (e < dk) { col = h * dk + e; dst = s_q + e; }
      else if (e < 2 * dk) { col = Hk + h * dk + e - dk; dst = s_k + e - dk; }
      else if (e < 2 * dk + 64) { col = 2 * Hk + h * p.dv + vb * 64 + e - 2 * dk; dst = s_v + e - 2 * dk; }
      else { col = 2 * Hk + Hv + h * p.dv + vb * 64 + e - 2 * dk - 64; dst = s_g + e - 2 * dk - 64; }
      const float* src = p.part + (size_t)row * p.N + p.col + col;
      float4 b[8], a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < 8; ++s) b[s] = s < p.slices ? __ldcg(reinterpret_cast<const float4*>(src + (size_t)s * p.M * p.N)) : a;
#pragma unroll
      for (int s = 0; s < 8; ++s) { a.x += b[s].x; a.y += b[s].y; a.z += b[s].z; a.w += b[s].w; }
      if (e < 2 * dk) a = rotated(p, a, pos, e < dk ? e : e - dk);
      const float sc = e >= dk && e < 2 * dk ? p.k_scale : 1.f;
      *reinterpret_cast<float4*>(dst) = make_float4(a.x * sc, a.y * sc, a.z * sc, a.w * sc);
    }
    __syncthreads();
    const float4 v = *reinterpret_cast<const float4*>(s_v + c);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const float kd = s_k[16 * i + grp], qd = s_q[16 * i + grp];
      S[i].x = fmaf(keep, S[i].x, kd * v.x); o.x = fmaf(S[i].x, qd, o.x);
      S[i].y = fmaf(keep, S[i].y, kd * v.y); o.y = fmaf(S[i].y, qd, o.y);
      S[i].z = fmaf(keep, S[i].z, kd * v.z); o.z = fmaf(S[i].z, qd, o.z);
      S[i].w = fmaf(keep, S[i].w, kd * v.w); o.w = fmaf(S[i].w, qd, o.w);
    }
    *reinterpret_cast<float4*>(&s_red[grp][c]) = o;
    __syncthreads();
    float y = 0.f;
    if (tid < 64) {
#pragma unroll
      for (int i = 0; i < 16; ++i) y += s_red[i][tid];
      const float ssq = warp_sum(y * y);
      if ((tid & 31) == 0) s_sum[tid >> 5] = ssq;
    }
    __syncthreads();
    float tot = s_sum[0] + s_sum[1];
    if (nvb > 1) {             // the head's other value blocks
      if (tid == 0) s_ssq = tot;
      cl.sync();
      tot = 0.f;
      for (int i = 0; i < nvb; ++i) tot += *cl.map_shared_rank(&s_ssq, i);
      cl.sync();
    }
    if (tid < 64) {
      const float r = p.mult / sqrtf(tot / (float)p.vdim + p.eps), z = s_g[tid];
      put(reinterpret_cast<T*>(p.out) + (size_t)row * p.ldo + h * p.dv + vb * 64 + tid, y * r * z / (1.f + expf(-z)));
    }
  }
#pragma unroll
  for (int i = 0; i < NS; ++i) *reinterpret_cast<float4*>(st + (size_t)(16 * i + grp) * p.dv) = S[i];
}

// ------------------------------------------------------------------ prompt segments
constexpr int CH = 128;              // rows of a chunk
constexpr int kSegWords = 4;
constexpr int kThreads = 256, kWarps = 8;

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - bf16_lo(hi), y - bf16_hi(hi));
}
// decay^n from its log2; n 0 is 1 whatever the decay
__device__ __forceinline__ float decayed(float lg, int n) { return n > 0 ? exp2f(lg * (float)n) : 1.f; }

// Shared tiles: blocks of `rows` x 64 columns, a row of 128 bytes whose 16-byte pieces are swizzled.
// Four columns c .. c + 3 of row r, as bf16 (LIMBS 2: and the rest in a second tile `lo_off` further)
template <int LIMBS>
__device__ __forceinline__ void put4(uint8_t* tile, uint32_t lo_off, int rows, int r, int c, const float4& v) {
  const uint32_t at = (uint32_t)((c >> 6) * rows * 128 + r * 128 + ((((c & 63) >> 3) ^ (r & 7)) << 4) + (c & 4) * 2);
  uint32_t h0, h1, l0, l1;
  split2(v.x, v.y, h0, l0);
  split2(v.z, v.w, h1, l1);
  *reinterpret_cast<uint2*>(tile + at) = make_uint2(h0, h1);
  if (LIMBS == 2) *reinterpret_cast<uint2*>(tile + lo_off + at) = make_uint2(l0, l1);
}

template <int KB, int VB>
struct Chunk {
  static constexpr int dk = KB * 64, DVB = VB * 64;
  static constexpr int K_LIMB = CH * dk * 2, V_BYTES = CH * DVB * 2, S_LIMB = dk * DVB * 2;
  static constexpr int SMEM = (2 * K_LIMB + V_BYTES > 2 * S_LIMB ? 2 * K_LIMB + V_BYTES : 2 * S_LIMB) + 1024;
  static_assert(SMEM <= 227 * 1024, "shared memory of one CTA");
};

// `cols` columns from `src` (rows `ld` apart) of `rows_all` rows into a shared tile; rows from `rows` on are zero.  ROT: rotated by
// the rows' positions from `pos` on, times `scale`, and with DECAY times decay^(rows - 1 - row).  Several loads in flight.
template <int LIMBS, bool ROT, bool DECAY>
__device__ __forceinline__ void stage(const RetentionParams& p, uint8_t* tile, uint32_t lo_off, const float* src, size_t ld, int rows_all, int cols,
                                      int rows, int pos, float scale, float lg) {
  constexpr int U = ROT ? 4 : 8;
  const int quads = cols / 4, n = rows_all * quads;
  for (int i0 = threadIdx.x; i0 < n; i0 += U * kThreads) {
    float4 x[U];
    float t[ROT ? U : 1][4];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * kThreads, r = i / quads, c = (i - r * quads) * 4;
      x[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < n && r < rows) x[u] = __ldcg(reinterpret_cast<const float4*>(src + r * ld + c));
      if constexpr (ROT) {
        t[u][0] = t[u][2] = 1.f;
        t[u][1] = t[u][3] = 0.f;
        const int k = c >> 1;
        const size_t at = (size_t)(pos + min(r, rows - 1)) * p.half + k;
        if (k < p.half) { t[u][0] = p.cos[at]; t[u][1] = p.sin[at]; }
        if (k + 1 < p.half) { t[u][2] = p.cos[at + 1]; t[u][3] = p.sin[at + 1]; }
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * kThreads, r = i / quads, c = (i - r * quads) * 4;
      if (i >= n) break;
      if constexpr (ROT) {
        const float f = DECAY ? scale * decayed(lg, rows - 1 - r) : scale;
        x[u] = make_float4((x[u].x * t[u][0] - x[u].y * t[u][1]) * f, (x[u].y * t[u][0] + x[u].x * t[u][1]) * f,
                           (x[u].z * t[u][2] - x[u].w * t[u][3]) * f, (x[u].w * t[u][2] + x[u].z * t[u][3]) * f);
      }
      put4<LIMBS>(tile, lo_off, rows_all, r, c, x[u]);
    }
  }
}

// keys and values of a chunk
template <int KB, int VB, bool DECAY>
__device__ __forceinline__ void stage_kv(const RetentionParams& p, uint8_t* k_s, uint8_t* v_s, int row0, int rows, int h, int vb, float lg) {
  using C = Chunk<KB, VB>;
  const int Hk = p.H * C::dk;
  const float* row = p.part + (size_t)row0 * p.N + p.col;
  stage<2, true, DECAY>(p, k_s, C::K_LIMB, row + Hk + h * C::dk, p.N, CH, C::dk, rows, p.pos[row0], p.k_scale, lg);
  stage<1, false, false>(p, v_s, 0, row + 2 * Hk + h * p.dv + vb * C::DVB, p.N, CH, C::DVB, rows, 0, 1.f, 0.f);
}

// grid (chunks of the longest segment, heads x value blocks, segments)
template <int KB, int VB>
__global__ void __launch_bounds__(kThreads) retention_kv_kernel(const RetentionParams p) {
  using C = Chunk<KB, VB>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* sp = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nvb = p.dv / C::DVB, h = blockIdx.y / nvb, vb = blockIdx.y % nvb, *seg = p.segs + blockIdx.z * kSegWords;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3, mi = lane >> 3;
  pdl_launch_dependents();
  pdl_wait();
  if ((int)blockIdx.x * CH >= seg[1]) return;
  const int row0 = seg[0] + blockIdx.x * CH, rows = min(CH, seg[1] - (int)blockIdx.x * CH);
  stage_kv<KB, VB, true>(p, sp, sp + 2 * C::K_LIMB, row0, rows, h, vb, p.decay[p.H + h]);
  __syncthreads();
  const uint32_t k_s = smem_u32(sp), v_s = k_s + 2 * C::K_LIMB;
  float* dst = p.kv + ((size_t)(seg[3] + blockIdx.x) * p.H + h) * C::dk * p.dv + vb * C::DVB;
  const int steps = (rows + 15) / 16;
  for (int item = warp; item < KB * 4 * VB; item += kWarps) {       // 16 key dims x 64 value columns
    const int mt = item / VB, nb = item % VB;
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    for (int kk = 0; kk < steps; ++kk) {
      uint32_t a[2][4];
      const int ra = 16 * kk + 8 * (mi >> 1) + (lane & 7), pc = 2 * (mt & 3) + (mi & 1);
      const uint32_t at = k_s + (mt >> 2) * CH * 128 + ra * 128 + ((pc ^ (ra & 7)) << 4);
      ldsm_x4_trans(at, a[0]);
      ldsm_x4_trans(at + C::K_LIMB, a[1]);
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        uint32_t b[4];
        const int rb = 16 * kk + 8 * (mi & 1) + (lane & 7);
        ldsm_x4_trans(v_s + nb * CH * 128 + rb * 128 + (((j + (mi >> 1)) ^ (rb & 7)) << 4), b);
#pragma unroll
        for (int l = 0; l < 2; ++l) {
          mma_bf16_16816(acc[j], a[l][0], a[l][1], a[l][2], a[l][3], b[0], b[1]);
          mma_bf16_16816(acc[j + 1], a[l][0], a[l][1], a[l][2], a[l][3], b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf)
        *reinterpret_cast<float2*>(dst + (size_t)(mt * 16 + g + 8 * hf) * p.dv + nb * 64 + 8 * j + 2 * t) = make_float2(acc[j][2 * hf], acc[j][2 * hf + 1]);
  }
}

// grid (quads of a state / 256, heads, segments): a chunk's sum is replaced by the state ahead of it
__global__ void __launch_bounds__(kThreads) retention_scan_kernel(const RetentionParams p) {
  const int h = blockIdx.y, *seg = p.segs + blockIdx.z * kSegWords, size = p.dk * p.dv;
  const int e = (blockIdx.x * kThreads + threadIdx.x) * 4;
  pdl_launch_dependents();
  pdl_wait();
  if (e >= size) return;
  const int rows = seg[1], nch = (rows + CH - 1) / CH;
  float4* st = reinterpret_cast<float4*>(p.state + ((size_t)seg[2] * p.H + h) * size + e);
  float4 S = p.pos[seg[0]] == 0 ? make_float4(0.f, 0.f, 0.f, 0.f) : *st;
  float* kv = p.kv + ((size_t)seg[3] * p.H + h) * size + e;
  const size_t next = (size_t)p.H * size;
  const float lg = p.decay[p.H + h], whole = decayed(lg, CH);
  for (int c0 = 0; c0 < nch; c0 += 8) {
    float4 add[8];
#pragma unroll
    for (int u = 0; u < 8; ++u)
      if (c0 + u < nch) add[u] = __ldcg(reinterpret_cast<const float4*>(kv + (c0 + u) * next));
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      if (c0 + u >= nch) break;
      *reinterpret_cast<float4*>(kv + (c0 + u) * next) = S;
      const int n = rows - (c0 + u) * CH;
      const float f = n >= CH ? whole : decayed(lg, n);
      S = make_float4(fmaf(f, S.x, add[u].x), fmaf(f, S.y, add[u].y), fmaf(f, S.z, add[u].z), fmaf(f, S.w, add[u].w));
    }
  }
  *st = S;
}

// grid (chunks of the longest segment, heads x value blocks, segments); a warp owns 16 rows
template <int KB, int VB>
__global__ void __launch_bounds__(kThreads) retention_chunk_kernel(const RetentionParams p) {
  using C = Chunk<KB, VB>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* sp = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nvb = p.dv / C::DVB, h = blockIdx.y / nvb, vb = blockIdx.y % nvb, *seg = p.segs + blockIdx.z * kSegWords;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3, mi = lane >> 3;
  pdl_launch_dependents();
  pdl_wait();
  if ((int)blockIdx.x * CH >= seg[1]) return;
  const int row0 = seg[0] + blockIdx.x * CH, rows = min(CH, seg[1] - (int)blockIdx.x * CH);
  const float lg = p.decay[p.H + h];
  const uint32_t base = smem_u32(sp);
  // this warp's queries as operand fragments, two limbs, through the shared tile
  const int lo_row = warp * 16;
  uint32_t q[2][KB * 4][4];
  stage<2, true, false>(p, sp, C::K_LIMB, p.part + (size_t)row0 * p.N + p.col + h * C::dk, p.N, CH, C::dk, rows, p.pos[row0], 1.f, 0.f);
  __syncthreads();
#pragma unroll
  for (int k = 0; k < KB * 4; ++k) {
    const int r = lo_row + 8 * (mi & 1) + (lane & 7);
    const uint32_t at = base + (k >> 2) * CH * 128 + r * 128 + (((2 * (k & 3) + (mi >> 1)) ^ (r & 7)) << 4);
    ldsm_x4(at, q[0][k]);
    ldsm_x4(at + C::K_LIMB, q[1][k]);
  }
  __syncthreads();
  // the state ahead of the chunk, two limbs
  const float* kv = p.kv + ((size_t)(seg[3] + blockIdx.x) * p.H + h) * C::dk * p.dv + vb * C::DVB;
  const bool zero = blockIdx.x == 0 && p.pos[seg[0]] == 0;
  if (!zero) stage<2, false, false>(p, sp, C::S_LIMB, kv, p.dv, C::dk, C::DVB, C::dk, 0, 1.f, 0.f);
  __syncthreads();
  float o[VB * 8][4];
#pragma unroll
  for (int j = 0; j < VB * 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  if (!zero && lo_row < rows) {
#pragma unroll
    for (int kk = 0; kk < KB * 4; ++kk) {
      const int rb = 16 * kk + 8 * (mi & 1) + (lane & 7);
#pragma unroll
      for (int j = 0; j < VB * 8; j += 2) {
        const uint32_t at = base + (j >> 3) * C::dk * 128 + rb * 128 + ((((j & 7) + (mi >> 1)) ^ (rb & 7)) << 4);
        uint32_t b[2][4];
        ldsm_x4_trans(at, b[0]);
        ldsm_x4_trans(at + C::S_LIMB, b[1]);
#pragma unroll
        for (int l = 0; l < 3; ++l) {        // hi hi, lo hi, hi lo
          const uint32_t(&a)[4] = q[l == 1][kk];
          const uint32_t(&s)[4] = b[l == 2];
          mma_bf16_16816(o[j], a[0], a[1], a[2], a[3], s[0], s[1]);
          mma_bf16_16816(o[j + 1], a[0], a[1], a[2], a[3], s[2], s[3]);
        }
      }
    }
    const float f0 = decayed(lg, lo_row + g + 1), f1 = decayed(lg, lo_row + g + 9);
#pragma unroll
    for (int j = 0; j < VB * 8; ++j) { o[j][0] *= f0; o[j][1] *= f0; o[j][2] *= f1; o[j][3] *= f1; }
  }
  __syncthreads();             // every warp is done with the state: keys and values take its place
  stage_kv<KB, VB, false>(p, sp, sp + 2 * C::K_LIMB, row0, rows, h, vb, lg);
  __syncthreads();
  if (lo_row >= rows) return;
  const uint32_t v_s = base + 2 * C::K_LIMB;
  for (int kt = 0; kt <= warp; ++kt) {       // 16 keys
    float s[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < KB * 2; ++kk)        // 32 dims
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int rk = kt * 16 + 8 * j + (lane & 7);
        const uint32_t at = base + (kk >> 1) * CH * 128 + rk * 128 + (((4 * (kk & 1) + mi) ^ (rk & 7)) << 4);
        uint32_t b[2][4];
        ldsm_x4(at, b[0]);
        ldsm_x4(at + C::K_LIMB, b[1]);
#pragma unroll
        for (int l = 0; l < 3; ++l)
#pragma unroll
          for (int w = 0; w < 2; ++w) {
            const uint32_t(&a)[4] = q[l == 1][2 * kk + w];
            mma_bf16_16816(s[j], a[0], a[1], a[2], a[3], b[l == 2][2 * w], b[l == 2][2 * w + 1]);
          }
      }
    uint32_t ph[4], pl[4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int away = lo_row + g + 8 * hf - (kt * 16 + 8 * j + 2 * t);
        const float x = away >= 0 ? s[j][2 * hf] * decayed(lg, away) : 0.f;
        const float y = away >= 1 ? s[j][2 * hf + 1] * decayed(lg, away - 1) : 0.f;
        split2(x, y, ph[2 * j + hf], pl[2 * j + hf]);
      }
    const int rb = kt * 16 + 8 * (mi & 1) + (lane & 7);
#pragma unroll
    for (int j = 0; j < VB * 8; j += 2) {
      uint32_t b[4];
      ldsm_x4_trans(v_s + (j >> 3) * CH * 128 + rb * 128 + ((((j & 7) + (mi >> 1)) ^ (rb & 7)) << 4), b);
      mma_bf16_16816(o[j], ph[0], ph[1], ph[2], ph[3], b[0], b[1]);
      mma_bf16_16816(o[j + 1], ph[0], ph[1], ph[2], ph[3], b[2], b[3]);
      mma_bf16_16816(o[j], pl[0], pl[1], pl[2], pl[3], b[0], b[1]);
      mma_bf16_16816(o[j + 1], pl[0], pl[1], pl[2], pl[3], b[2], b[3]);
    }
  }
  const int Hv = p.H * p.dv;
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int r = lo_row + g + 8 * hf;
    if (p.raw) {
      if (r >= rows) continue;
      float* dst = p.raw + (size_t)(row0 + r) * Hv + h * p.dv + vb * C::DVB + 2 * t;
#pragma unroll
      for (int j = 0; j < VB * 8; ++j) *reinterpret_cast<float2*>(dst + 8 * j) = make_float2(o[j][2 * hf], o[j][2 * hf + 1]);
      continue;
    }
    float ssq = 0.f;
#pragma unroll
    for (int j = 0; j < VB * 8; ++j) ssq += o[j][2 * hf] * o[j][2 * hf] + o[j][2 * hf + 1] * o[j][2 * hf + 1];
    ssq += __shfl_xor_sync(0xffffffffu, ssq, 1);
    ssq += __shfl_xor_sync(0xffffffffu, ssq, 2);
    if (r >= rows) continue;
    const float f = p.mult / sqrtf(ssq / (float)p.vdim + p.eps);
    const float* z = p.part + (size_t)(row0 + r) * p.N + p.col + 2 * p.H * C::dk + Hv + h * p.dv + 2 * t;
    __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)(row0 + r) * p.ldo + h * p.dv + 2 * t;
#pragma unroll
    for (int j = 0; j < VB * 8; ++j) {
      const float2 zz = __ldcg(reinterpret_cast<const float2*>(z + 8 * j));
      *reinterpret_cast<uint32_t*>(dst + 8 * j) =
          pack_bf16(o[j][2 * hf] * f * zz.x / (1.f + __expf(-zz.x)), o[j][2 * hf + 1] * f * zz.y / (1.f + __expf(-zz.y)));
    }
  }
}

// a warp per (row, head); grid (rows, heads / 8)
__global__ void __launch_bounds__(kThreads) retention_out_kernel(const RetentionParams p) {
  const int row = blockIdx.x, h = blockIdx.y * kWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31, Hv = p.H * p.dv;
  pdl_launch_dependents();
  pdl_wait();
  if (h >= p.H) return;
  const float* o = p.raw + (size_t)row * Hv + h * p.dv;
  float ssq = 0.f;
  for (int c = lane * 4; c < p.dv; c += 128) {
    const float4 x = __ldcg(reinterpret_cast<const float4*>(o + c));
    ssq += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
  }
  const float f = p.mult / sqrtf(warp_sum(ssq) / (float)p.vdim + p.eps);
  const float* z = p.part + (size_t)row * p.N + p.col + 2 * p.H * p.dk + Hv + h * p.dv;
  __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + (size_t)row * p.ldo + h * p.dv;
  for (int c = lane * 4; c < p.dv; c += 128) {
    const float4 x = __ldcg(reinterpret_cast<const float4*>(o + c)), y = __ldcg(reinterpret_cast<const float4*>(z + c));
    *reinterpret_cast<uint2*>(dst + c) = make_uint2(pack_bf16(x.x * f * silu(y.x), x.y * f * silu(y.y)), pack_bf16(x.z * f * silu(y.z), x.w * f * silu(y.w)));
  }
}

template <int KB, typename T>
int launch_step(const RetentionParams& p, cudaStream_t st) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.dv / 64, p.H, p.M);
  cfg.blockDim = dim3(256);
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = p.dv / 64;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  static const bool no_pdl = getenv("B2_NO_PDL") != nullptr;  // measurement switch, as in b2_launch
  cfg.numAttrs = no_pdl ? 1 : 2;
  return (int)cudaLaunchKernelEx(&cfg, retention_step_kernel<KB, T>, p);
}

template <typename T>
int launch_steps(const RetentionParams& p, cudaStream_t st) {
  switch (p.dk / 64) {
    case 1: return launch_step<1, T>(p, st);
    case 2: return launch_step<2, T>(p, st);
    case 3: return launch_step<3, T>(p, st);
    case 4: return launch_step<4, T>(p, st);
    case 6: return launch_step<6, T>(p, st);
    case 8: return launch_step<8, T>(p, st);
  }
  return -1;
}

int value_block(int dk, int dv) { return dk <= 128 && dv % 128 == 0 ? 2 : 1; }      // blocks of 64 value dims per CTA

template <int KB, int VB>
int launch_segments(RetentionParams p, int n_segs, int most, cudaStream_t st) {
  using C = Chunk<KB, VB>;
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(retention_kv_kernel<KB, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(retention_chunk_kernel<KB, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM);
    if (e != cudaSuccess) return (int)e;
    configured[dev & 63] = true;
  }
  const int nvb = p.dv / C::DVB;
  if (nvb == 1) p.raw = nullptr;
  const dim3 grid(most, p.H * nvb, n_segs);
  int rc = b2_launch(retention_kv_kernel<KB, VB>, grid, dim3(kThreads), C::SMEM, st, true, p);
  if (!rc) rc = b2_launch(retention_scan_kernel, dim3((p.dk * p.dv / 4 + kThreads - 1) / kThreads, p.H, n_segs), dim3(kThreads), 0, st, true, p);
  if (!rc) rc = b2_launch(retention_chunk_kernel<KB, VB>, grid, dim3(kThreads), C::SMEM, st, true, p);
  if (!rc && nvb > 1) rc = b2_launch(retention_out_kernel, dim3(p.M, (p.H + kWarps - 1) / kWarps), dim3(kThreads), 0, st, true, p);
  return rc;
}

bool retention_ok(const RetentionParams& p) {
  return p.M >= 1 && p.slices >= 1 && p.slices <= 8 && p.H >= 1 && p.dk % 64 == 0 && p.dk >= 64 && p.dv % 64 == 0 && p.dv >= 64 && p.dv <= 512 &&
         p.col >= 0 && p.col % 4 == 0 && p.N % 4 == 0 && p.col + 2 * p.H * (p.dk + p.dv) <= p.N && p.half >= 0 && 2 * p.half <= p.dk &&
         (!p.half || (p.cos && p.sin)) && p.vdim >= 1 && p.ldo >= p.H * p.dv && p.ldo % 4 == 0;
}

}  // namespace

// part: fp32 [slices][M][N], columns col .. as in RetentionParams; decay [2][H] (decay, log2 of it); cos / sin [positions][half].
extern "C" int b2_retention_step(const float* part, int slices, int M, int N, int col, int H, int dk, int dv, int vdim, const int* req,
                                 const int* pos, const float* cos, const float* sin, int half, float k_scale, float eps, float mult,
                                 const float* decay, float* state, void* out, int ldo, int f32, void* stream) {
  RetentionParams p = {};
  p.part = part; p.slices = slices; p.M = M; p.N = N; p.col = col; p.H = H; p.dk = dk; p.dv = dv; p.vdim = vdim; p.req = req; p.pos = pos;
  p.cos = cos; p.sin = sin; p.half = half; p.k_scale = k_scale; p.eps = eps; p.mult = mult; p.decay = decay; p.state = state; p.out = out; p.ldo = ldo;
  if (!retention_ok(p) || M > 65535) return -1;
  return f32 ? launch_steps<float>(p, (cudaStream_t)stream) : launch_steps<__nv_bfloat16>(p, (cudaStream_t)stream);
}

// 1 when the tensor-core form covers the sizes; b2_retention_raw: it wants `raw`
extern "C" int b2_retention_chunks_ok(int dk, int dv) { return dk % 64 == 0 && dv % 64 == 0 && dk >= 64 && dk <= 256 && dv >= 64 && dv <= 512; }
extern "C" int b2_retention_raw(int dk, int dv) { return dv > 64 * value_block(dk, dv); }
extern "C" int b2_retention_chunk_rows() { return CH; }

// Prompt segments, one slice: segs [n_segs][4], `most` chunks in the longest one; kv: fp32 [chunks][H][dk][dv]; out in bf16.
extern "C" int b2_retention_segments(const float* part, int M, int N, int col, int H, int dk, int dv, int vdim, const int* pos, const int* segs,
                                     int n_segs, int most, const float* cos, const float* sin, int half, float k_scale, float eps, float mult,
                                     const float* decay, float* state, float* kv, float* raw, void* out, int ldo, void* stream) {
  RetentionParams p = {};
  p.part = part; p.slices = 1; p.M = M; p.N = N; p.col = col; p.H = H; p.dk = dk; p.dv = dv; p.vdim = vdim; p.pos = pos;
  p.cos = cos; p.sin = sin; p.half = half; p.k_scale = k_scale; p.eps = eps; p.mult = mult; p.decay = decay; p.state = state; p.out = out; p.ldo = ldo;
  p.segs = segs; p.kv = kv; p.raw = raw;
  if (!retention_ok(p) || !b2_retention_chunks_ok(dk, dv) || n_segs < 1 || n_segs > 65535 || most < 1 || !segs || !kv) return -1;
  const int vb = value_block(dk, dv);
  if (dv > 64 * vb && !raw) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  switch (dk / 64 * 10 + vb) {
    case 11: return launch_segments<1, 1>(p, n_segs, most, st);
    case 12: return launch_segments<1, 2>(p, n_segs, most, st);
    case 21: return launch_segments<2, 1>(p, n_segs, most, st);
    case 22: return launch_segments<2, 2>(p, n_segs, most, st);
    case 31: return launch_segments<3, 1>(p, n_segs, most, st);
    case 41: return launch_segments<4, 1>(p, n_segs, most, st);
  }
  return -3;
}

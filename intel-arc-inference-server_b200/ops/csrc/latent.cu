// Latent attention: queries and keys / values go through low-rank latents, and a token's cache entry is its key-value
// latent c and one rotated key part shared by all heads -- [page][16][lc], lc = kvp + rp (both padded to 64).
//
//   latent_prep_kernel    folds the down projection's slices, RMS norm of the query latent and of c, rotation of the
//                         shared key part, append to the page pool
//   latent_absorb_kernel  decode form of the queries: rotated part, and q_nope through W_uk per head, so that scores
//                         are taken against c itself -- [row][head][lc]
//   latent_rows_kernel    split-KV attention of decode rows over c (mma.m16n8k16): a CTA serves 16 or 32 heads of one row,
//                         whose keys and values are the same tiles (64 keys, tiled TMA copies of 16 keys x 64 dims)
//   latent_simple_kernel  the same in plain fp32 arithmetic for either element type: models served in 32-bit, and shapes
//                         outside the tensor-core kernels
//   latent_merge_kernel   merge of the splits, and the value up projection W_uv of the merged latent
//   latent_gather_kernel, latent_rope_q_kernel   prompt form (keys and values expanded by GEMMs, attn_prefill.cu):
//                         cache rows of the segments' keys into contiguous rows; rotation of the queries
//
// Angles, norms, scores, softmax weights and sums are fp32; the softmax weights enter their product as two bf16 limbs.
// Rows are described by three int arrays (request slot, position, token), which the control block of a decode step
// holds at fixed offsets and a mixed batch has in a table of its own.
#include "common.cuh"

#include <mutex>
#include <unordered_map>

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
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
  const uint32_t v = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(bf16_lo(v), bf16_hi(v));
}

struct Rows {            // one entry per row of the step
  const int* req;
  const int* pos;
};
struct Rope {            // tables [max_pos][dims / 2]
  const float* cos_t;
  const float* sin_t;
  int dims;
};

// element i of a rotated vector: rotate-half pairs (i, i + dims / 2) on the first `dims` elements
__device__ __forceinline__ float rope_at(const float* v, int i, int pos, const Rope& r) {
  const int half = r.dims >> 1;
  if (i >= r.dims) return v[i];
  const int j = i < half ? i : i - half;
  const float c = r.cos_t[(size_t)pos * half + j], s = r.sin_t[(size_t)pos * half + j];
  return i < half ? v[i] * c - v[i + half] * s : v[i] * c + v[i - half] * s;
}

// ------------------------------------------------------------------ down projection -> latents, cache append
struct PrepParams {
  const float* part;     // [S][M][qp + kvp + rp]
  int S, M, q_rank, qp, kv_rank, kvp, rot, rp;
  const float *q_norm, *kv_norm;
  float eps;
  Rows rows;
  const int* block_table;
  int max_blocks;
  Rope rope;
  void* cq;              // [M][qp]
  void* cache;           // [page][16][kvp + rp]
};

constexpr int kRopeShared = 128;    // angle pairs kept in shared memory

template <typename T>
__global__ void __launch_bounds__(512) latent_prep_kernel(const PrepParams p) {
  extern __shared__ __align__(16) float v[];       // the row's qp + kvp + rp values
  __shared__ float red[2][16];
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float s_cos[kRopeShared], s_sin[kRopeShared];
  const int m = blockIdx.x, n = p.qp + p.kvp + p.rp, tid = threadIdx.x, nw = blockDim.x >> 5;
  const int pos = p.rows.pos[m], req = p.rows.req[m];
  float sq = 0.f, sc = 0.f;
  for (int i = tid * 4; i < n; i += blockDim.x * 4) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b[8];
#pragma unroll
    for (int s = 0; s < 8; ++s)          // every slice's value requested before the first is used (S <= 8)
      b[s] = s < p.S ? __ldcg(reinterpret_cast<const float4*>(p.part + ((size_t)s * p.M + m) * n + i)) : a;
#pragma unroll
    for (int s = 0; s < 8; ++s) { a.x += b[s].x; a.y += b[s].y; a.z += b[s].z; a.w += b[s].w; }
    *reinterpret_cast<float4*>(v + i) = a;
    const float q = a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;   // padding columns are zero
    if (i < p.qp) sq += q;
    else if (i < p.qp + p.kvp) sc += q;
  }
  // the page and the angles while the slices arrive
  const int page = p.block_table[(size_t)req * p.max_blocks + (pos >> 4)], half = p.rope.dims >> 1;
  Rope rope = p.rope;
  int rope_pos = pos;
  if (half <= kRopeShared) {
    for (int i = tid; i < half; i += blockDim.x) {
      s_cos[i] = p.rope.cos_t[(size_t)pos * half + i];
      s_sin[i] = p.rope.sin_t[(size_t)pos * half + i];
    }
    rope.cos_t = s_cos;
    rope.sin_t = s_sin;
    rope_pos = 0;
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sc; }
  __syncthreads();
  sq = sc = 0.f;
  for (int i = 0; i < nw; ++i) { sq += red[0][i]; sc += red[1][i]; }
  const float rq = 1.f / sqrtf(sq / (float)p.q_rank + p.eps), rc = 1.f / sqrtf(sc / (float)p.kv_rank + p.eps);
  const int lc = p.kvp + p.rp;
  T* cq = reinterpret_cast<T*>(p.cq) + (size_t)m * p.qp;
  for (int i = tid; i < p.qp; i += blockDim.x) cq[i] = from_f<T>(i < p.q_rank ? v[i] * rq * p.q_norm[i] : 0.f);
  T* dst = reinterpret_cast<T*>(p.cache) + ((size_t)page * 16 + (pos & 15)) * lc;
  for (int i = tid; i < lc; i += blockDim.x) {
    float o = 0.f;
    if (i < p.kv_rank) o = v[p.qp + i] * rc * p.kv_norm[i];
    else if (i >= p.kvp && i - p.kvp < p.rot) o = rope_at(v + p.qp + p.kvp, i - p.kvp, rope_pos, rope);
    dst[i] = from_f<T>(o);
  }
}

// ------------------------------------------------------------------ queries against the latent
// grid (head, kvp / 128, row groups of 8); 256 threads = 4 slices of the head's dims x 64 pairs of latent dims
struct AbsorbParams {
  const float* q;        // [S][M][H * (dn + rp)]
  int S, M, H, dn, rp, rot, kvp;
  const void* w_uk;      // [H * dn][kvp]
  Rows rows;
  Rope rope;
  void* out;             // [M][H][kvp + rp]
};

template <typename T>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const AbsorbParams p) {
  extern __shared__ float sm[];           // q [8][dn + rp], then partial sums [4][8][128]
  const int h = blockIdx.x, r0 = blockIdx.y * 128, m0 = blockIdx.z * 8, mt = min(8, p.M - m0);
  const int dk = p.dn + p.rp, lc = p.kvp + p.rp, tid = threadIdx.x;
  float* qs = sm;
  float* red = sm + 8 * dk;
  const int sl = tid >> 6, r = r0 + (tid & 63) * 2, per = p.dn / 4;
  const T* w = reinterpret_cast<const T*>(p.w_uk) + ((size_t)h * p.dn + sl * per) * p.kvp + r;
  float2 wv[16];           // the first weights do not wait for the queries
  if (r < p.kvp) {
#pragma unroll
    for (int u = 0; u < 16; ++u) wv[u] = load2(w + (size_t)u * p.kvp);
  }
  pdl_launch_dependents();
  pdl_wait();
  for (int i = tid; i < 8 * dk; i += 256) {
    const int m = i / dk, d = i - m * dk;
    float a = 0.f;
    if (m < mt)
      for (int s = 0; s < p.S; ++s) a += p.q[((size_t)s * p.M + m0 + m) * p.H * dk + (size_t)h * dk + d];
    qs[i] = a;
  }
  __syncthreads();
  float acc[8][2];
#pragma unroll
  for (int m = 0; m < 8; ++m) acc[m][0] = acc[m][1] = 0.f;
  if (r < p.kvp) {
    const float* q = qs + sl * per;
    for (int d = 0; d < per; d += 16) {      // dn is a multiple of 64
#pragma unroll
      for (int m = 0; m < 8; ++m)
        if (m < mt) {
#pragma unroll
          for (int u = 0; u < 16; ++u) {
            const float qv = q[m * dk + d + u];
            acc[m][0] = fmaf(qv, wv[u].x, acc[m][0]);
            acc[m][1] = fmaf(qv, wv[u].y, acc[m][1]);
          }
        }
      if (d + 16 < per) {
#pragma unroll
        for (int u = 0; u < 16; ++u) wv[u] = load2(w + (size_t)(d + 16 + u) * p.kvp);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < 8; ++m) {
    red[(sl * 8 + m) * 128 + (tid & 63) * 2] = acc[m][0];
    red[(sl * 8 + m) * 128 + (tid & 63) * 2 + 1] = acc[m][1];
  }
  __syncthreads();
  for (int i = tid; i < mt * 128; i += 256) {
    const int m = i >> 7, c = i & 127;
    if (r0 + c >= p.kvp) continue;
    const float o = ((red[m * 128 + c] + red[(8 + m) * 128 + c]) + red[(16 + m) * 128 + c]) + red[(24 + m) * 128 + c];
    reinterpret_cast<T*>(p.out)[((size_t)(m0 + m) * p.H + h) * lc + r0 + c] = from_f<T>(o);
  }
  if (blockIdx.y == 0)
    for (int i = tid; i < mt * p.rp; i += 256) {
      const int m = i / p.rp, c = i - m * p.rp;
      const float o = c < p.rot ? rope_at(qs + m * dk + p.dn, c, p.rows.pos[m0 + m], p.rope) : 0.f;
      reinterpret_cast<T*>(p.out)[((size_t)(m0 + m) * p.H + h) * lc + p.kvp + c] = from_f<T>(o);
    }
}

// ------------------------------------------------------------------ decode attention over the latent (tensor cores)
struct RowsParams {
  CUtensorMap map;         // the layer's cache as a matrix [pages * 16][lc]; boxes of 16 rows x 64 columns
  const __nv_bfloat16* q;  // [M][H][lc]
  float* o_part;           // [M][H][nsplit][kvp]
  float* ml_part;          // [M][H][nsplit][2]
  Rows rows;
  const int* block_table;
  int max_blocks, H, kvp, lc, nsplit, window;   // window 0: every earlier position
  float scale_log2;
};

constexpr int KT = 64;             // keys per tile
constexpr int kRowsThreads = 256;

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
// byte offset of (row, dim d) in a tile kept as 64-dim blocks of R rows x 128 bytes with the 128-byte swizzle
template <int R>
__device__ __forceinline__ uint32_t tile_off(int row, int d) {
  return (uint32_t)((d >> 6) * (R * 128) + row * 128 + ((((d & 63) >> 3) ^ (row & 7)) << 4));
}

// keys [lo, hi) of a split: the row's visible pages in nsplit equal parts
__device__ __forceinline__ void split_range(int pos, int window, int nsplit, int split, int& lo, int& hi) {
  const int first = window > 0 ? max(0, pos - window + 1) : 0;
  const int page0 = first >> 4, pages = (pos >> 4) + 1 - page0, pps = (pages + nsplit - 1) / nsplit;
  lo = (page0 + split * pps) * 16;
  hi = min(pos + 1, lo + pps * 16);
}

// MT: tiles of 16 heads per CTA; KVC: blocks of 64 latent dims; QREG: the queries' fragments stay in registers (one head
// tile, one block of rotated dims), which saves each warp reading them from shared memory again for every tile.  Scores: the eight warps are MT head tiles x 8 / MT slices of the tile's keys; product
// with the values: MT head tiles x 8 / MT slices of the latent's dims.  The weights pass between the two through shared
// memory as bf16 limbs (hi + lo).  Two tiles of keys in flight.
template <int MT, int KVC, bool QREG>
__global__ void __launch_bounds__(kRowsThreads, 1) latent_rows_kernel(const __grid_constant__ RowsParams p) {
  constexpr int QR = MT * 16, NSL = 8 / MT, KSL = KT / NSL, NJ = KSL / 8;
  constexpr int NT = KVC * MT, DW = NT * 8;        // this warp's slice of the latent's dims: NT groups of 8
  extern __shared__ uint8_t smem_raw[];
  __shared__ float s_mx[QR][NSL];
  const int nc = p.lc >> 6;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t q_s = base, kv_s = q_s + nc * QR * 128, kvB = nc * KT * 128;
  const uint32_t ph_s = kv_s + 2 * kvB, pl_s = ph_s + QR * 128, bar0 = pl_s + QR * 128;
  const int m = blockIdx.x, split = blockIdx.y, h0 = blockIdx.z * QR;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int mt = warp % MT, sl = warp / MT;
  if (tid == 0) {
    mbar_init(bar0, 1);
    mbar_init(bar0 + 8, 1);
    mbar_fence_init();
    prefetch_tmap(&p.map);
  }
  pdl_launch_dependents();
  pdl_wait();
  const int pos = p.rows.pos[m], req = p.rows.req[m];
  int key0, key1;
  split_range(pos, p.window, p.nsplit, split, key0, key1);
  const int klo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int ntile = key1 > key0 ? (key1 - key0 + KT - 1) / KT : 0;
  const int* bt = p.block_table + (size_t)req * p.max_blocks;
  __syncthreads();
  auto issue = [&](int i) {          // warp 0: tile i into buffer i & 1; pages past the split repeat its last page
    const uint32_t dst = kv_s + (i & 1) * kvB, bar = bar0 + 8 * (i & 1);
    const int pg0 = (key0 >> 4) + i * (KT / 16), pg_last = (key1 - 1) >> 4;
    if (lane == 0) mbar_expect_tx(bar, kvB);
    __syncwarp();
    for (int j = lane; j < nc * (KT / 16); j += 32) {
      const int pi = j & 3, c = j >> 2;
      tma_load_2d(dst + c * (KT * 128) + pi * 2048, &p.map, c * 64, bt[min(pg0 + pi, pg_last)] * 16, bar);
    }
  };
  if (warp == 0) {
    if (ntile > 0) issue(0);
    if (ntile > 1) issue(1);
  }
  {
    // the queries: a batch of vectors per thread requested before the first is stored
    const int vpr = p.lc / 8, total = min(QR, p.H - h0) * vpr;
    constexpr int B = 6;
    for (int i0 = tid; i0 < QR * vpr; i0 += B * kRowsThreads) {
      uint4 x[B];
#pragma unroll
      for (int u = 0; u < B; ++u) {       // rows of one (row, head group) are contiguous
        const int i = i0 + u * kRowsThreads;
        x[u] = i < total ? __ldcg(reinterpret_cast<const uint4*>(p.q + ((size_t)m * p.H + h0) * p.lc) + i) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
      for (int u = 0; u < B; ++u) {
        const int i = i0 + u * kRowsThreads, r = i / vpr, v = i - r * vpr;
        if (i < QR * vpr)
          asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};" ::"r"(q_s + tile_off<QR>(r, v * 8)), "r"(x[u].x), "r"(x[u].y), "r"(x[u].z),
                       "r"(x[u].w)
                       : "memory");
      }
    }
  }
  __syncthreads();

  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, lsum[2] = {0.f, 0.f};
  // ldmatrix lanes: a block of 64 dims keeps a row's 16-byte pieces at (piece XOR row mod 8), so a lane's address in it
  // is a base plus one of eight swizzled offsets that do not change from block to block
  const uint32_t qrow = q_s + (mt * 16 + (lane & 15)) * 128, qsw = lane & 7, qhi = lane >> 4;
  const uint32_t krow = (sl * KSL + (lane & 7)) * 128, kmi = lane >> 3;
  uint32_t qa[QREG ? KVC + 1 : 1][4][4];
  if (QREG) {
#pragma unroll
    for (int c = 0; c < KVC + 1; ++c)
#pragma unroll
      for (int k = 0; k < 4; ++k)
        ldsm_x4(qrow + c * (QR * 128) + (((2 * k + qhi) ^ qsw) << 4), qa[c][k][0], qa[c][k][1], qa[c][k][2], qa[c][k][3]);
  }
  bool ok = true;
  for (int i = 0; i < ntile; ++i) {
    const uint32_t kt = kv_s + (i & 1) * kvB;
    if (ok) ok = mbar_wait(bar0 + 8 * (i & 1), (i >> 1) & 1, ERR_ATTN_WAIT);
    // ---- scores of this warp's heads x keys: per block of 64 dims all operands first, then four independent chains
    float s[4][NJ][4];
#pragma unroll
    for (int c = 0; c < 4; ++c)
#pragma unroll
      for (int j = 0; j < NJ; ++j) s[c][j][0] = s[c][j][1] = s[c][j][2] = s[c][j][3] = 0.f;
    auto block = [&](int c, const uint32_t (&a)[4][4]) {
      uint32_t b[NJ][2][4];
#pragma unroll
      for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int k = 0; k < 2; ++k)
          ldsm_x4(kt + c * (KT * 128) + krow + j * 1024 + (((4 * k + kmi) ^ qsw) << 4), b[j][k][0], b[j][k][1], b[j][k][2], b[j][k][3]);
#pragma unroll
      for (int k = 0; k < 4; ++k)
#pragma unroll
        for (int j = 0; j < NJ; ++j)
          mma_bf16_16816(s[k][j], a[k][0], a[k][1], a[k][2], a[k][3], b[j][k >> 1][2 * (k & 1)], b[j][k >> 1][2 * (k & 1) + 1]);
    };
    if constexpr (QREG) {
#pragma unroll
      for (int c = 0; c < KVC + 1; ++c) block(c, qa[c]);
    } else {
#pragma unroll 2
      for (int c = 0; c < nc; ++c) {
        uint32_t a[4][4];
#pragma unroll
        for (int k = 0; k < 4; ++k)
          ldsm_x4(qrow + c * (QR * 128) + (((2 * k + qhi) ^ qsw) << 4), a[k][0], a[k][1], a[k][2], a[k][3]);
        block(c, a);
      }
    }
    float mnew[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int key = key0 + i * KT + sl * KSL + 8 * j + 2 * t + (e & 1);
        const float v = key < key1 && key >= klo ? ((s[0][j][e] + s[1][j][e]) + (s[2][j][e] + s[3][j][e])) * p.scale_log2 : -INFINITY;
        s[0][j][e] = v;
        mnew[e >> 1] = fmaxf(mnew[e >> 1], v);
      }
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      mnew[hf] = fmaxf(mnew[hf], __shfl_xor_sync(0xffffffffu, mnew[hf], 1));
      mnew[hf] = fmaxf(mnew[hf], __shfl_xor_sync(0xffffffffu, mnew[hf], 2));
      if (t == 0) s_mx[mt * 16 + g + 8 * hf][sl] = mnew[hf];
    }
    __syncthreads();     // maxima of every slice; every warp is done with tile i - 1
    if (warp == 0 && i > 0 && i + 1 < ntile) issue(i + 1);
    float corr[2];
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      float v = mx[hf];
#pragma unroll
      for (int q = 0; q < NSL; ++q) v = fmaxf(v, s_mx[mt * 16 + g + 8 * hf][q]);
      corr[hf] = v == -INFINITY ? 1.f : exp2f(mx[hf] - v);
      lsum[hf] *= corr[hf];
      mx[hf] = v;
    }
#pragma unroll
    for (int j = 0; j < NJ; ++j)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        float pe[2], lo[2];
        uint32_t hi;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          pe[e] = mx[hf] == -INFINITY ? 0.f : exp2f(s[0][j][2 * hf + e] - mx[hf]);
          lsum[hf] += pe[e];
        }
        hi = pack_bf16(pe[0], pe[1]);
        lo[0] = pe[0] - bf16_lo(hi);
        lo[1] = pe[1] - bf16_hi(hi);
        const uint32_t off = tile_off<QR>(mt * 16 + g + 8 * hf, sl * KSL + 8 * j) + 4 * t;
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(ph_s + off), "r"(hi) : "memory");
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(pl_s + off), "r"(pack_bf16(lo[0], lo[1])) : "memory");
      }
    __syncthreads();
    // ---- O += P C over this warp's dims
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      o[j][0] *= corr[0]; o[j][1] *= corr[0]; o[j][2] *= corr[1]; o[j][3] *= corr[1];
    }
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      uint32_t ph[4], pl[4];
      const uint32_t off = (mt * 16 + (lane & 15)) * 128 + (((2 * kk + qhi) ^ qsw) << 4);
      ldsm_x4(ph_s + off, ph[0], ph[1], ph[2], ph[3]);
      ldsm_x4(pl_s + off, pl[0], pl[1], pl[2], pl[3]);
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        const int mi = lane >> 3, d = sl * DW + 8 * min(j + (mi >> 1), NT - 1);
        uint32_t b[4];
        ldsm_x4_trans(kt + (d >> 6) * (KT * 128) + (16 * kk + 8 * (mi & 1) + (lane & 7)) * 128 + ((((uint32_t)(d & 63) >> 3) ^ qsw) << 4),
                      b[0], b[1], b[2], b[3]);
        mma_bf16_16816(o[j], ph[0], ph[1], ph[2], ph[3], b[0], b[1]);
        if (j + 1 < NT) mma_bf16_16816(o[j + 1], ph[0], ph[1], ph[2], ph[3], b[2], b[3]);
        mma_bf16_16816(o[j], pl[0], pl[1], pl[2], pl[3], b[0], b[1]);
        if (j + 1 < NT) mma_bf16_16816(o[j + 1], pl[0], pl[1], pl[2], pl[3], b[2], b[3]);
      }
    }
  }
  // ---- the split's partials: O against the running maximum, (maximum, sum)
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    lsum[hf] += __shfl_xor_sync(0xffffffffu, lsum[hf], 1);
    lsum[hf] += __shfl_xor_sync(0xffffffffu, lsum[hf], 2);
  }
  __syncthreads();
#pragma unroll
  for (int hf = 0; hf < 2; ++hf)
    if (t == 0) s_mx[mt * 16 + g + 8 * hf][sl] = lsum[hf];
  __syncthreads();
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int h = h0 + mt * 16 + g + 8 * hf;
    if (h >= p.H) continue;
    const size_t row = ((size_t)m * p.H + h) * p.nsplit + split;
    if (sl == 0 && t == 0) {
      float l = 0.f;
#pragma unroll
      for (int q = 0; q < NSL; ++q) l += s_mx[mt * 16 + g + 8 * hf][q];
      p.ml_part[2 * row] = mx[hf];
      p.ml_part[2 * row + 1] = l;
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
      *reinterpret_cast<float2*>(p.o_part + row * p.kvp + sl * DW + 8 * j + 2 * t) = make_float2(o[j][2 * hf], o[j][2 * hf + 1]);
  }
}

// ------------------------------------------------------------------ the same in plain fp32 arithmetic
struct SimpleParams {
  const void* cache;       // [pages * 16][lc]
  const void* q;           // [M][H][lc]
  float *o_part, *ml_part; // nsplit = 1
  Rows rows;
  const int* block_table;
  int max_blocks, H, kvp, lc, window;
  float scale;
};
constexpr int kSimpleDims = 16;    // latent dims per thread: kvp <= 2048

template <typename T>
__global__ void __launch_bounds__(128) latent_simple_kernel(const SimpleParams p) {
  extern __shared__ float qs[];      // [lc]
  __shared__ float sc[128];
  __shared__ size_t row_of[128];
  pdl_launch_dependents();
  pdl_wait();
  const int m = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos = p.rows.pos[m];
  const int* bt = p.block_table + (size_t)p.rows.req[m] * p.max_blocks;
  const T* cache = reinterpret_cast<const T*>(p.cache);
  for (int i = tid; i < p.lc; i += 128) qs[i] = to_f(reinterpret_cast<const T*>(p.q)[((size_t)m * p.H + h) * p.lc + i]);
  float o[kSimpleDims];
#pragma unroll
  for (int i = 0; i < kSimpleDims; ++i) o[i] = 0.f;
  float mx = -INFINITY, l = 0.f;
  for (int k0 = p.window > 0 ? max(0, pos - p.window + 1) : 0; k0 <= pos; k0 += 128) {
    const int n = min(128, pos + 1 - k0);
    __syncthreads();
    if (tid < n) row_of[tid] = ((size_t)bt[(k0 + tid) >> 4] * 16 + ((k0 + tid) & 15)) * p.lc;
    __syncthreads();
    for (int j = warp; j < n; j += 4) {
      const T* c = cache + row_of[j];
      float s = 0.f;
      for (int d = lane; d < p.lc; d += 32) s = fmaf(qs[d], to_f(c[d]), s);
      s = warp_sum(s);
      if (lane == 0) sc[j] = s * p.scale;
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
      const T* c = cache + row_of[j];
#pragma unroll
      for (int i = 0; i < kSimpleDims; ++i)
        if (tid + 128 * i < p.kvp) o[i] = fmaf(w, to_f(c[tid + 128 * i]), o[i]);
    }
  }
  const size_t row = (size_t)m * p.H + h;
#pragma unroll
  for (int i = 0; i < kSimpleDims; ++i)
    if (tid + 128 * i < p.kvp) p.o_part[row * p.kvp + tid + 128 * i] = o[i];
  if (tid == 0) {
    p.ml_part[2 * row] = mx * 1.4426950408889634f;    // the merge works in powers of two
    p.ml_part[2 * row + 1] = l;
  }
}

// ------------------------------------------------------------------ merge of the splits + value up projection
// grid (head, dv / 16, row groups of 8), 256 threads: the rows' merged latents in shared memory (every CTA of a head
// merges them for itself: the partials come from L2), then a warp per two value dims, whose weights are requested before
// the kernel waits for its predecessor
struct MergeParams {
  const float *o_part, *ml_part;
  int M, H, nsplit, kvp, dv;
  const void* w_uv;      // [H * dv][kvp]
  void* out;             // [M][ld], head h at column h * dv
  int ld;
};

// eight consecutive values
struct Raw8f { float4 a, b; };
__device__ __forceinline__ void fetch8(const float* p, Raw8f& r) {
  r.a = __ldg(reinterpret_cast<const float4*>(p));
  r.b = __ldg(reinterpret_cast<const float4*>(p) + 1);
}
__device__ __forceinline__ void fetch8(const __nv_bfloat16* p, uint4& r) { r = __ldg(reinterpret_cast<const uint4*>(p)); }
__device__ __forceinline__ void expand8(const Raw8f& r, float (&v)[8]) {
  v[0] = r.a.x; v[1] = r.a.y; v[2] = r.a.z; v[3] = r.a.w; v[4] = r.b.x; v[5] = r.b.y; v[6] = r.b.z; v[7] = r.b.w;
}
__device__ __forceinline__ void expand8(const uint4& r, float (&v)[8]) {
  v[0] = bf16_lo(r.x); v[1] = bf16_hi(r.x); v[2] = bf16_lo(r.y); v[3] = bf16_hi(r.y);
  v[4] = bf16_lo(r.z); v[5] = bf16_hi(r.z); v[6] = bf16_lo(r.w); v[7] = bf16_hi(r.w);
}
template <typename T> struct Raw8 { using type = uint4; };
template <> struct Raw8<float> { using type = Raw8f; };

template <typename T>
__global__ void __launch_bounds__(256) latent_merge_kernel(const MergeParams p) {
  extern __shared__ __align__(16) float lat[];          // [8][kvp], then the partial merges of split groups [G - 1][mt][kvp]
  __shared__ float wt[8][64];
  const int h = blockIdx.x, m0 = blockIdx.z * 8, mt = min(8, p.M - m0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, v0 = blockIdx.y * 16 + warp * 2;
  typename Raw8<T>::type raw[2][2];
  const T* w = reinterpret_cast<const T*>(p.w_uv) + ((size_t)h * p.dv + v0) * p.kvp;
#pragma unroll
  for (int d = 0; d < 2; ++d)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = i * 256 + lane * 8;
      if (r < p.kvp) fetch8(w + (size_t)d * p.kvp + r, raw[d][i]);
    }
  pdl_launch_dependents();
  pdl_wait();
  if (warp < mt) {      // nsplit <= 64: two splits per lane
    const float* ml = p.ml_part + ((size_t)(m0 + warp) * p.H + h) * p.nsplit * 2;
    float mx[2], l[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = lane + 32 * i;
      mx[i] = s < p.nsplit ? ml[2 * s] : -INFINITY;
      l[i] = s < p.nsplit ? ml[2 * s + 1] : 0.f;
    }
    const float top = warp_max(fmaxf(mx[0], mx[1]));
    float e[2], sum = 0.f;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      e[i] = mx[i] == -INFINITY ? 0.f : exp2f(mx[i] - top);
      sum += e[i] * l[i];
    }
    const float inv = 1.f / warp_sum(sum);
#pragma unroll
    for (int i = 0; i < 2; ++i) wt[warp][lane + 32 * i] = e[i] * inv;
  }
  __syncthreads();
  const int vecs = mt * p.kvp / 4;
  int G = 1;                         // groups of threads that share the splits of few rows
  while (G < 8 && 2 * G * vecs <= 256 && 2 * G <= p.nsplit) G *= 2;
  const int per = (p.nsplit + G - 1) / G;
  for (int u = tid; u < G * vecs; u += 256) {
    const int grp = u / vecs, i = (u - grp * vecs) * 4, m = i / p.kvp, r = i - m * p.kvp;
    const int s_lo = grp * per, s_hi = min(p.nsplit, s_lo + per);
    const float* o = p.o_part + ((size_t)(m0 + m) * p.H + h) * p.nsplit * p.kvp + r;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s0 = s_lo; s0 < s_hi; s0 += 16) {
      float4 v[16];
#pragma unroll
      for (int q = 0; q < 16; ++q)
        v[q] = s0 + q < s_hi ? __ldcg(reinterpret_cast<const float4*>(o + (size_t)(s0 + q) * p.kvp)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int q = 0; q < 16; ++q) {
        const float x = s0 + q < s_hi ? wt[m][s0 + q] : 0.f;
        a.x = fmaf(x, v[q].x, a.x); a.y = fmaf(x, v[q].y, a.y); a.z = fmaf(x, v[q].z, a.z); a.w = fmaf(x, v[q].w, a.w);
      }
    }
    *reinterpret_cast<float4*>(lat + (grp ? (size_t)8 * p.kvp + (size_t)(grp - 1) * mt * p.kvp : 0) + i) = a;
  }
  __syncthreads();
  if (G > 1) {
    for (int i = tid; i < mt * p.kvp; i += 256) {
      float a = lat[i];
      for (int q = 1; q < G; ++q) a += lat[8 * p.kvp + (q - 1) * mt * p.kvp + i];
      lat[i] = a;
    }
    __syncthreads();
  }
  float acc[2][8];
#pragma unroll
  for (int m = 0; m < 8; ++m) acc[0][m] = acc[1][m] = 0.f;
  auto accumulate = [&](int r, const typename Raw8<T>::type& r0, const typename Raw8<T>::type& r1) {
    float w0[8], w1[8];
    expand8(r0, w0);
    expand8(r1, w1);
#pragma unroll
    for (int m = 0; m < 8; ++m)
      if (m < mt) {
        float x[8];
        *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(lat + m * p.kvp + r);
        *reinterpret_cast<float4*>(x + 4) = *reinterpret_cast<const float4*>(lat + m * p.kvp + r + 4);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          acc[0][m] = fmaf(w0[j], x[j], acc[0][m]);
          acc[1][m] = fmaf(w1[j], x[j], acc[1][m]);
        }
      }
  };
#pragma unroll
  for (int i = 0; i < 2; ++i)
    if (i * 256 + lane * 8 < p.kvp) accumulate(i * 256 + lane * 8, raw[0][i], raw[1][i]);
  for (int r = 512 + lane * 8; r < p.kvp; r += 256) {
    typename Raw8<T>::type r0, r1;
    fetch8(w + r, r0);
    fetch8(w + p.kvp + r, r1);
    accumulate(r, r0, r1);
  }
#pragma unroll
  for (int m = 0; m < 8; ++m)
    if (m < mt) {
      const float a = warp_sum(acc[0][m]), b = warp_sum(acc[1][m]);
      if (lane == 0) {
        T* dst = reinterpret_cast<T*>(p.out) + (size_t)(m0 + m) * p.ld + (size_t)h * p.dv + v0;
        dst[0] = from_f<T>(a);
        dst[1] = from_f<T>(b);
      }
    }
}

// ------------------------------------------------------------------ prompt form: keys of the segments, queries
// one CTA per key row: c and the rotated part of (slot, position) into contiguous rows
__global__ void __launch_bounds__(96) latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, const int* __restrict__ kreq,
                                                           const int* __restrict__ kpos, const int* __restrict__ block_table,
                                                           int max_blocks, int kvp, int rp, __nv_bfloat16* __restrict__ c,
                                                           __nv_bfloat16* __restrict__ kr) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, pos = kpos[r];
  const int page = block_table[(size_t)kreq[r] * max_blocks + (pos >> 4)];
  const uint4* src = reinterpret_cast<const uint4*>(cache + ((size_t)page * 16 + (pos & 15)) * (kvp + rp));
  for (int i = threadIdx.x; i < (kvp + rp) / 8; i += blockDim.x) {
    const uint4 v = src[i];
    if (i < kvp / 8) reinterpret_cast<uint4*>(c + (size_t)r * kvp)[i] = v;
    else reinterpret_cast<uint4*>(kr + (size_t)r * rp)[i - kvp / 8] = v;
  }
}

// one CTA per row: rotates dims dn .. dn + rot of every head in place
__global__ void __launch_bounds__(256) latent_rope_q_kernel(__nv_bfloat16* __restrict__ q, const int* __restrict__ pos_of, int H,
                                                            int dn, int rp, const Rope rope) {
  pdl_launch_dependents();
  pdl_wait();
  const int half = rope.dims >> 1, pos = pos_of[blockIdx.x];
  __nv_bfloat16* row = q + (size_t)blockIdx.x * H * (dn + rp) + dn;
  for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
    const int h = i / half, j = i - h * half;
    __nv_bfloat16* a = row + (size_t)h * (dn + rp) + j;
    const float c = rope.cos_t[(size_t)pos * half + j], s = rope.sin_t[(size_t)pos * half + j];
    const float u = __bfloat162float(a[0]), v = __bfloat162float(a[half]);
    a[0] = __float2bfloat16(u * c - v * s);
    a[half] = __float2bfloat16(v * c + u * s);
  }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeTiledFn encode_fn() {
  static EncodeTiledFn fn = nullptr;
  if (!fn) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres) == cudaSuccess &&
        qres == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeTiledFn>(ptr);
  }
  return fn;
}

int rows_smem(int mt, int lc) { return 1024 + (lc / 64) * (mt * 16 + 2 * KT) * 128 + 2 * mt * 16 * 128 + 32; }

template <int MT, int KVC, bool QREG>
int launch_rows_kernel(const RowsParams& p, int M, cudaStream_t st) {
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(latent_rows_kernel<MT, KVC, QREG>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024 - 4096);
    if (e != cudaSuccess) return (int)e;
    configured[dev & 63] = true;
  }
  return b2_launch(latent_rows_kernel<MT, KVC, QREG>, dim3(M, p.nsplit, (p.H + MT * 16 - 1) / (MT * 16)), dim3(kRowsThreads),
                   rows_smem(MT, p.lc), st, true, p);
}

template <int MT, int KVC>
int launch_rows_form(const RowsParams& p, int M, cudaStream_t st) {
  if constexpr (MT == 1)
    if (p.lc == p.kvp + 64) return launch_rows_kernel<MT, KVC, true>(p, M, st);
  return launch_rows_kernel<MT, KVC, false>(p, M, st);
}

template <int MT>
int launch_rows(const RowsParams& p, int M, cudaStream_t st) {
  switch (p.kvp / 64) {
    case 1: return launch_rows_form<MT, 1>(p, M, st);
    case 2: return launch_rows_form<MT, 2>(p, M, st);
    case 3: return launch_rows_form<MT, 3>(p, M, st);
    case 4: return launch_rows_form<MT, 4>(p, M, st);
    case 5: return launch_rows_form<MT, 5>(p, M, st);
    case 6: return launch_rows_form<MT, 6>(p, M, st);
    case 7: return launch_rows_form<MT, 7>(p, M, st);
    case 8: return launch_rows_form<MT, 8>(p, M, st);
  }
  return -1;
}

template <typename F>
int set_smem(F* fn, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  if (bytes > 200 * 1024) return -5;
  return (int)cudaFuncSetAttribute(fn, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

}  // namespace

extern "C" int b2_latent_prep(const float* part, int S, int M, int q_rank, int qp, int kv_rank, int kvp, int rot, int rp,
                              const float* q_norm, const float* kv_norm, float eps, const int* req, const int* pos,
                              const int* block_table, int max_blocks, const float* cos_t, const float* sin_t, int rope_dims,
                              void* cq, void* cache, int f32, void* stream) {
  if (M < 1 || S < 1 || S > 8 || qp % 64 || kvp % 64 || rp % 64 || rope_dims % 2 || rope_dims > rot || rot > rp) return -1;
  PrepParams p{part, S, M, q_rank, qp, kv_rank, kvp, rot, rp, q_norm, kv_norm, eps, {req, pos}, block_table, max_blocks,
               {cos_t, sin_t, rope_dims}, cq, cache};
  const size_t smem = (size_t)(qp + kvp + rp) * 4;
  if (smem > 48 * 1024) return -5;
  return f32 ? b2_launch(latent_prep_kernel<float>, dim3(M), dim3(512), smem, (cudaStream_t)stream, true, p)
             : b2_launch(latent_prep_kernel<__nv_bfloat16>, dim3(M), dim3(512), smem, (cudaStream_t)stream, true, p);
}

extern "C" int b2_latent_absorb(const float* q, int S, int M, int H, int dn, int rp, int rot, int kvp, const void* w_uk,
                                const int* pos, const float* cos_t, const float* sin_t, int rope_dims, void* out, int f32,
                                void* stream) {
  if (M < 1 || M > 8 * 65535 || dn % 64 || rp % 64 || kvp % 64 || rope_dims > rot || rot > rp) return -1;
  AbsorbParams p{q, S, M, H, dn, rp, rot, kvp, w_uk, {nullptr, pos}, {cos_t, sin_t, rope_dims}, out};
  const size_t smem = (size_t)(8 * (dn + rp) + 4 * 8 * 128) * 4;
  if (smem > 48 * 1024) return -5;
  const dim3 grid(H, (kvp + 127) / 128, (M + 7) / 8);
  return f32 ? b2_launch(latent_absorb_kernel<float>, grid, dim3(256), smem, (cudaStream_t)stream, true, p)
             : b2_launch(latent_absorb_kernel<__nv_bfloat16>, grid, dim3(256), smem, (cudaStream_t)stream, true, p);
}

// 1 when the tensor-core decode kernel covers the shape
extern "C" int b2_latent_rows_ok(int H, int kvp, int rp) {
  return kvp % 64 == 0 && rp % 64 == 0 && kvp <= 512 && rows_smem(H > 16 ? 2 : 1, kvp + rp) <= 227 * 1024 - 4096;
}

// q [M][H][kvp + rp], cache [num_pages][16][kvp + rp] bf16 -> partials of nsplit splits
extern "C" int b2_latent_rows(const void* q, const void* cache, int num_pages, int M, int H, int kvp, int rp, const int* req,
                              const int* pos, const int* block_table, int max_blocks, float* o_part, float* ml_part,
                              int nsplit, int window, float scale, void* stream) {
  if (M < 1 || nsplit < 1 || nsplit > 64 || !b2_latent_rows_ok(H, kvp, rp)) return -1;
  RowsParams p;
  EncodeTiledFn fn = encode_fn();
  if (!fn) return -100;
  const int lc = kvp + rp;
  cuuint64_t dims[2] = {(cuuint64_t)lc, (cuuint64_t)num_pages * 16};
  cuuint64_t strides[1] = {(cuuint64_t)lc * 2};
  cuuint32_t box[2] = {64, 16}, estr[2] = {1, 1};
  CUresult r = fn(&p.map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(cache), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return -101 - (int)r;
  p.q = (const __nv_bfloat16*)q; p.o_part = o_part; p.ml_part = ml_part; p.rows = {req, pos};
  p.block_table = block_table; p.max_blocks = max_blocks; p.H = H; p.kvp = kvp; p.lc = lc; p.nsplit = nsplit;
  p.window = window > 0 ? window : 0; p.scale_log2 = scale * 1.4426950408889634f;
  // two head tiles per CTA halve the cache reads; a step too small to fill half the GPU that way takes one
  const bool pair = H > 16 && M * nsplit * ((H + 31) / 32) > 74;
  return pair ? launch_rows<2>(p, M, (cudaStream_t)stream) : launch_rows<1>(p, M, (cudaStream_t)stream);
}

extern "C" int b2_latent_simple(const void* q, const void* cache, int M, int H, int kvp, int rp, const int* req, const int* pos,
                                const int* block_table, int max_blocks, float* o_part, float* ml_part, int window, float scale,
                                int f32, void* stream) {
  if (M < 1 || kvp > 128 * kSimpleDims) return -1;
  SimpleParams p{cache, q, o_part, ml_part, {req, pos}, block_table, max_blocks, H, kvp, kvp + rp, window > 0 ? window : 0, scale};
  const size_t smem = (size_t)(kvp + rp) * 4;
  return f32 ? b2_launch(latent_simple_kernel<float>, dim3(M, H), dim3(128), smem, (cudaStream_t)stream, true, p)
             : b2_launch(latent_simple_kernel<__nv_bfloat16>, dim3(M, H), dim3(128), smem, (cudaStream_t)stream, true, p);
}

extern "C" int b2_latent_merge(const float* o_part, const float* ml_part, int M, int H, int nsplit, int kvp, int dv,
                               const void* w_uv, void* out, int ld, int f32, void* stream) {
  if (M < 1 || M > 8 * 65535 || nsplit < 1 || nsplit > 64 || kvp % 64 || dv % 64) return -1;
  MergeParams p{o_part, ml_part, M, H, nsplit, kvp, dv, w_uv, out, ld};
  const size_t smem = (size_t)8 * kvp * 4 + 4096;     // split groups only form where they share at most 1024 values
  const dim3 grid(H, dv / 16, (M + 7) / 8);
  int rc = f32 ? set_smem(latent_merge_kernel<float>, smem) : set_smem(latent_merge_kernel<__nv_bfloat16>, smem);
  if (rc) return rc;
  return f32 ? b2_launch(latent_merge_kernel<float>, grid, dim3(256), smem, (cudaStream_t)stream, true, p)
             : b2_launch(latent_merge_kernel<__nv_bfloat16>, grid, dim3(256), smem, (cudaStream_t)stream, true, p);
}

extern "C" int b2_latent_gather(const void* cache, const int* kreq, const int* kpos, int n, const int* block_table,
                                int max_blocks, int kvp, int rp, void* c, void* kr, void* stream) {
  if (n < 1 || kvp % 64 || rp % 64) return -1;
  return b2_launch(latent_gather_kernel, dim3(n), dim3(96), 0, (cudaStream_t)stream, true, (const __nv_bfloat16*)cache, kreq,
                   kpos, block_table, max_blocks, kvp, rp, (__nv_bfloat16*)c, (__nv_bfloat16*)kr);
}

extern "C" int b2_latent_rope_q(void* q, const int* pos, int M, int H, int dn, int rp, const float* cos_t, const float* sin_t,
                                int rope_dims, void* stream) {
  if (M < 1 || rope_dims > rp) return -1;
  Rope r{cos_t, sin_t, rope_dims};
  return b2_launch(latent_rope_q_kernel, dim3(M), dim3(256), 0, (cudaStream_t)stream, true, (__nv_bfloat16*)q, pos, H, dn, rp,
                   r);
}

B2_DEFINE_STATUS(latent)

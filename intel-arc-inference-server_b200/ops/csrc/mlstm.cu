// Matrix-memory recurrence with exponential gates (mLSTM): per head a state S [dk][dv], a normaliser n [dk] and a running
// maximum m, all fp32, one block per (slot, head, 32 value dims); every block has its own copy of n and m.
//
//   m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' likewise with k alone
//   o  = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6)          q scaled by dim^-1/2
//   i  = cap tanh(z_i / cap),  f = logsigmoid(cap tanh(z_f / cap))
//   out = o / rms(o) * norm * sigmoid(z_g)                  rms over the head's value dims
//
//   mlstm_step_kernel   rows in order, one token at a time: a cluster of dv / 64 CTAs per (sequence, head) folds the
//                       projection's slices, updates the state and writes the gated output; either element type
//   mlstm_gates_kernel  prompt segments: gates of all rows, and the running maximum at every chunk of 64 rows
//   mlstm_scan_kernel   prompt segments: a CTA walks the chunks of one (segment, head, 32 value dims) on the tensor cores
//   mlstm_out_kernel    prompt segments: head norm and output gate
//
// Chunk form.  With F_t the sum of f over the chunk's rows up to t, a_s = i_s - F_s and M_t = max(m0, max_{s <= t} a_s):
//     m_t = F_t + M_t;   P[t][s] = e^(a_s - M_t) (k_s . q_t), s <= t
//     o_t = (e^(m0 - M_t) S0^T q_t + sum_s P[t][s] v_s) / (max(|e^(m0 - M_t) n0 . q_t + sum_s P[t][s]|, e^(-m_t)) + 1e-6)
//     S <- e^(m0 - M) S0 + sum_s e^(a_s - M) k_s v_s^T        (M of the last row)
// so every exponent is at most 0.  Queries, keys and values are the projection's bf16; P, the state and the weighted values
// enter their products as two bf16 limbs.
//
// A sequence's first row (position 0) starts from a zero state whatever its slot holds.
#include "common.cuh"

#include <cooperative_groups.h>

using namespace b2;
namespace cg = cooperative_groups;

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) {
  const float x = cap * tanhf(z / cap);
  return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}
constexpr int VB = 32;                                                                // value dims of a state block
__host__ __device__ constexpr int state_block(int dk) { return dk * (VB + 1) + 4; }   // S [dk][32], n [dk], m, padding

// ------------------------------------------------------------------ one token at a time
struct StepParams {
  const float* part;      // [slices][M][N]: q [H dk] | k [H dk] | v [H dv] | g [H dv] | i [H] | f [H] | padding
  int slices, M, N, H, dk, dv, vdim;
  const int *req, *pos;
  const float* gate_bias; // [2 H]
  float cap, q_scale, eps;
  const float* norm;      // [H dv], padding 0
  float* state;           // [slots][H][dv / 32][state_block]
  void* out;              // [M][H dv]
};

// KB: blocks of 64 key dims.  256 threads: 16 groups of 4 value columns x 16 groups of key dims (d = 16 i + group)
template <int KB, typename T>
__global__ void __launch_bounds__(256) mlstm_step_kernel(const StepParams p) {
  constexpr int dk = KB * 64, NS = KB * 4, NN = (dk + 255) / 256;
  __shared__ __align__(16) float s_q[dk], s_k[dk], s_v[64], s_g[64], s_red[16][64], s_sum[8], s_gate[2];
  __shared__ float s_ssq;
  const int vb = blockIdx.x, nvb = gridDim.x, h = blockIdx.y, row0 = blockIdx.z;
  const int tid = threadIdx.x, grp = tid >> 4, c = (tid & 15) * 4;
  pdl_launch_dependents();
  pdl_wait();
  const int slot = p.req[row0];
  if (row0 > 0 && p.req[row0 - 1] == slot) return;        // the whole cluster leaves: another CTA walks this sequence
  constexpr int SB = state_block(dk);
  float* blk = p.state + (((size_t)slot * p.H + h) * nvb + vb) * 2 * SB;      // two blocks per CTA
  float* st = blk + (c >> 5) * SB + (c & 31);
  float4 S[NS];
  float n[NN], m = 0.f;
  const bool fresh = p.pos[row0] == 0;
#pragma unroll
  for (int i = 0; i < NS; ++i)
    S[i] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : __ldcg(reinterpret_cast<const float4*>(st + (16 * i + grp) * VB));
#pragma unroll
  for (int i = 0; i < NN; ++i) {
    const int d = tid + 256 * i;
    n[i] = fresh || d >= dk ? 0.f : __ldcg(blk + dk * VB + d);
  }
  if (!fresh) m = __ldcg(blk + SB - 4);
  const int Hk = p.H * dk, Hv = p.H * p.dv;
  cg::cluster_group cl = cg::this_cluster();
  for (int row = row0; row < p.M && p.req[row] == slot; ++row) {
    __syncthreads();            // the row before is done with the shared rows
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
      float4 b[8], a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < 8; ++s)
        b[s] = s < p.slices ? __ldcg(reinterpret_cast<const float4*>(p.part + ((size_t)s * p.M + row) * p.N + col)) : a;
#pragma unroll
      for (int s = 0; s < 8; ++s) { a.x += b[s].x; a.y += b[s].y; a.z += b[s].z; a.w += b[s].w; }
      const float sc = e < dk ? p.q_scale : 1.f;
      *reinterpret_cast<float4*>(dst) = make_float4(a.x * sc, a.y * sc, a.z * sc, a.w * sc);
    }
    if (tid >= 254) {          // the two gates
      const int w = tid - 254, col = 2 * Hk + 2 * Hv + w * p.H + h;
      float z = 0.f;
      for (int s = 0; s < p.slices; ++s) z += __ldcg(p.part + ((size_t)s * p.M + row) * p.N + col);
      z += p.gate_bias[w * p.H + h];
      s_gate[w] = w ? log_forget_gate(z, p.cap) : log_input_gate(z, p.cap);
    }
    __syncthreads();
    const float li = s_gate[0], lf = s_gate[1], mn = fmaxf(lf + m, li);
    const float keep = expf(lf + m - mn), add = expf(li - mn);
    m = mn;
    float nq = 0.f;
#pragma unroll
    for (int i = 0; i < NN; ++i) {
      const int d = tid + 256 * i;
      if (d < dk) {
        n[i] = fmaf(keep, n[i], add * s_k[d]);
        nq = fmaf(n[i], s_q[d], nq);
      }
    }
    nq = warp_sum(nq);
    if ((tid & 31) == 0) s_sum[tid >> 5] = nq;
    const float4 v = *reinterpret_cast<const float4*>(s_v + c);
    const float4 av = make_float4(add * v.x, add * v.y, add * v.z, add * v.w);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const float kd = s_k[16 * i + grp], qd = s_q[16 * i + grp];
      S[i].x = fmaf(keep, S[i].x, kd * av.x); o.x = fmaf(S[i].x, qd, o.x);
      S[i].y = fmaf(keep, S[i].y, kd * av.y); o.y = fmaf(S[i].y, qd, o.y);
      S[i].z = fmaf(keep, S[i].z, kd * av.z); o.z = fmaf(S[i].z, qd, o.z);
      S[i].w = fmaf(keep, S[i].w, kd * av.w); o.w = fmaf(S[i].w, qd, o.w);
    }
    *reinterpret_cast<float4*>(&s_red[grp][c]) = o;
    __syncthreads();
    float y = 0.f, ssq = 0.f;
    if (tid < 64) {
      float a = 0.f, q = 0.f;
#pragma unroll
      for (int i = 0; i < 16; ++i) a += s_red[i][tid];
#pragma unroll
      for (int i = 0; i < 8; ++i) q += s_sum[i];
      y = a / (fmaxf(fabsf(q), expf(-m)) + 1e-6f);
      ssq = warp_sum(y * y);
    }
    __syncthreads();
    if (tid < 64 && (tid & 31) == 0) s_sum[tid >> 5] = ssq;
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
      const int col = h * p.dv + vb * 64 + tid;
      const float r = 1.f / sqrtf(tot / (float)p.vdim + p.eps);
      put(reinterpret_cast<T*>(p.out) + (size_t)row * Hv + col, y * r * p.norm[col] / (1.f + expf(-s_g[tid])));
    }
  }
#pragma unroll
  for (int i = 0; i < NS; ++i) *reinterpret_cast<float4*>(st + (16 * i + grp) * VB) = S[i];
#pragma unroll
  for (int i = 0; i < NN; ++i)
    if (tid + 256 * i < dk) blk[dk * VB + tid + 256 * i] = blk[SB + dk * VB + tid + 256 * i] = n[i];
  if (tid < 2) blk[tid * SB + SB - 4] = m;
}

// ------------------------------------------------------------------ prompt segments
constexpr int CH = 64;               // rows of a chunk
constexpr int kSegWords = 4;         // first row, rows, slot, first chunk (counted over all segments)
constexpr int kGateBlock = 4 * CH;   // per (head, chunk): a_s, M_t (both times log2 e), m_t of the rows; m0 (times log2 e)
constexpr float kLog2e = 1.4426950408889634f;
__device__ __forceinline__ float exp2_fast(float x) {      // subnormal results are zero
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct GatesParams {
  const float* z;         // [rows][ldz]: z_i [H] | z_f [H]
  int ldz, H, dk, nvb, chunks;
  const int *segs, *pos;
  const float* gate_bias;
  float cap;
  const float* state;
  float* gates;           // [H][chunks][kGateBlock]
};

// grid (heads, segments), a warp per chunk: sums and maxima inside the chunks, the chunks' m0 in order, then the rows
__global__ void __launch_bounds__(256) mlstm_gates_kernel(const GatesParams p) {
  extern __shared__ float sm[];       // per chunk: sum of f, max of a; then m0
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, *seg = p.segs + blockIdx.y * kSegWords;
  const int row0 = seg[0], rows = seg[1], slot = seg[2], nch = (rows + CH - 1) / CH;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* out = p.gates + ((size_t)h * p.chunks + seg[3]) * kGateBlock;
  const float bi = p.gate_bias[h], bf = p.gate_bias[p.H + h];
  for (int c = warp; c < nch; c += 8) {
    float f[2], a[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = c * CH + 2 * lane + e;
      f[e] = 0.f;
      a[e] = -INFINITY;
      if (r < rows) {
        const float* z = p.z + (size_t)(row0 + r) * p.ldz + h;
        f[e] = log_forget_gate(z[p.H] + bf, p.cap);
        a[e] = log_input_gate(z[0] + bi, p.cap);
      }
    }
    float run = f[0] + f[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += v;
    }
    const float F0 = run - f[1], F1 = run;
    a[0] -= F0;
    a[1] -= F1;
    float top = fmaxf(a[0], a[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, top, o);
      if (lane >= o) top = fmaxf(top, v);
    }
    float before = __shfl_up_sync(0xffffffffu, top, 1);
    if (lane == 0) before = -INFINITY;
    float* g = out + (size_t)c * kGateBlock;
    *reinterpret_cast<float2*>(g + 2 * lane) = make_float2(a[0] * kLog2e, a[1] * kLog2e);
    *reinterpret_cast<float2*>(g + CH + 2 * lane) = make_float2(fmaxf(before, a[0]), top);     // without m0 yet
    *reinterpret_cast<float2*>(g + 2 * CH + 2 * lane) = make_float2(F0, F1);
    if (lane == 31) {
      sm[2 * c] = run;
      sm[2 * c + 1] = top;
    }
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    float m = p.pos[row0] == 0 ? 0.f : p.state[((size_t)slot * p.H + h) * p.nvb * state_block(p.dk) + state_block(p.dk) - 4];
    for (int c = 0; c < nch; ++c) {
      const float next = sm[2 * c] + fmaxf(m, sm[2 * c + 1]);
      sm[2 * c] = m;
      m = next;
    }
  }
  __syncthreads();
  for (int c = warp; c < nch; c += 8) {
    float* g = out + (size_t)c * kGateBlock;
    const float m0 = sm[2 * c];
    float2 M = *reinterpret_cast<float2*>(g + CH + 2 * lane), F = *reinterpret_cast<float2*>(g + 2 * CH + 2 * lane);
    M.x = fmaxf(M.x, m0);
    M.y = fmaxf(M.y, m0);
    *reinterpret_cast<float2*>(g + CH + 2 * lane) = make_float2(M.x * kLog2e, M.y * kLog2e);
    *reinterpret_cast<float2*>(g + 2 * CH + 2 * lane) = make_float2(F.x + M.x, F.y + M.y);
    if (lane == 0) g[3 * CH] = m0 * kLog2e;
  }
}

struct ScanParams {
  CUtensorMap map;        // the projection [rows][N]: q | k | v | g; boxes of 64 rows x 64 columns
  const int *segs, *pos;
  int H, dv, chunks;
  float q_scale_log2;
  const float* gates;
  float* state;
  float* o;               // [rows][H dv], before the head norm
};

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
// byte offset of a 16-byte piece (8 bf16) of a row of 128 bytes, 128-byte swizzle
__device__ __forceinline__ uint32_t piece(int row, int pc) { return (uint32_t)(row * 128 + ((pc ^ (row & 7)) << 4)); }

constexpr int kScanWork = 256, kScanThreads = kScanWork + 32;     // eight working warps and one that fetches

template <int KB>
struct Scan {
  static constexpr int BLK = CH * 128;                       // 64 rows x 64 dims
  static constexpr int OFF_K = KB * BLK, OFF_V = 2 * KB * BLK, OFF_G = OFF_V + BLK;
  static constexpr int STAGE = OFF_G + kGateBlock * 4;
  static constexpr int NST = KB <= 2 ? 3 : 2;                // chunks in flight
  static constexpr int OFF_P = NST * STAGE;                  // P as two limbs, of two chunks
  static constexpr int OFF_NT = OFF_P + 4 * BLK;             // n's limbs, of two chunks
  static constexpr int OFF_X = OFF_NT + 2 * KB * 1024;       // partial read-outs [8 warps][4 row groups][2][32 lanes][4]
  static constexpr int OFF_F = OFF_X + 8 * 4 * 1024;         // row sums of P [2 chunks][2][64], n . q [2][64], b [2 chunks][64]
                                                             // (fp32), b's limbs [2 chunks][2][64] (bf16)
  static constexpr int OFF_BAR = OFF_F + 10 * CH * 4;
  static constexpr int SMEM = OFF_BAR + 32 + 1024;
  static_assert(SMEM <= 227 * 1024, "shared memory of one CTA");
};

// Eight warps.  The state is S^T [32 value columns][dk] in MMA accumulators for the whole walk: warp = (tile of 16 value
// columns, quarter of the key dims).  Products are written with the value dimension as M, so accumulators become A operands
// in registers; the quarters' read-outs meet in shared memory, each warp finishing 16 of the chunk's 64 rows.  For the
// products with the keys a warp owns 16 rows and every second group of 16 keys up to them; n . q are products with two more
// key rows, n's bf16 limbs.  Between two barriers the warps read out and update the state for one chunk and make the next
// chunk's P, which does not depend on the state.  A ninth warp fetches.
template <int KB>
__global__ void __launch_bounds__(kScanThreads) mlstm_scan_kernel(const __grid_constant__ ScanParams p) {
  using L = Scan<KB>;
  constexpr int dk = KB * 64;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* sp = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t base = smem_u32(sp), bar0 = base + L::OFF_BAR;
  float* s_sum = reinterpret_cast<float*>(sp + L::OFF_F);
  float *s_nq = s_sum + 4 * CH, *s_b = s_nq + 2 * CH;
  __nv_bfloat16* s_bl = reinterpret_cast<__nv_bfloat16*>(s_b + 2 * CH);
  const int vb = blockIdx.x, nvb = gridDim.x, h = blockIdx.y, *seg = p.segs + blockIdx.z * kSegWords;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int vt = warp & 1, dq = warp >> 1;              // state: value tile, quarter of the key dims
  const int rt = warp >> 1, ke = warp & 1;              // scores: row tile, parity of the key groups
  if (tid == 0) {
    for (int i = 0; i < L::NST; ++i) mbar_init(bar0 + 8 * i, 1);
    mbar_fence_init();
    prefetch_tmap(&p.map);
  }
  pdl_launch_dependents();
  pdl_wait();
  const int row0 = seg[0], rows = seg[1], slot = seg[2], nch = (rows + CH - 1) / CH;
  const float* gates = p.gates + ((size_t)h * p.chunks + seg[3]) * kGateBlock;
  float* st_g = p.state + (((size_t)slot * p.H + h) * nvb + vb) * state_block(dk);
  const bool fresh = p.pos[row0] == 0;
  __syncthreads();
  auto stage = [](int c) { return c % L::NST; };
  auto arrived = [&](int c) { return mbar_wait(bar0 + 8 * stage(c), (c / L::NST) & 1, ERR_GDN_WAIT); };
  bool ok = true;
  if (warp == 8) {
    auto fetch = [&](int c) {
      const uint32_t dst = base + stage(c) * L::STAGE, bar = bar0 + 8 * stage(c);
      const int y = row0 + c * CH;
      mbar_expect_tx(bar, L::STAGE);
#pragma unroll
      for (int b = 0; b < KB; ++b) {
        tma_load_2d(dst + b * L::BLK, &p.map, h * dk + b * 64, y, bar);
        tma_load_2d(dst + L::OFF_K + b * L::BLK, &p.map, (p.H + h) * dk + b * 64, y, bar);
      }
      tma_load_2d(dst + L::OFF_V, &p.map, 2 * p.H * dk + h * p.dv + (vb >> 1) * 64, y, bar);
      bulk_g2s(dst + L::OFF_G, gates + (size_t)c * kGateBlock, kGateBlock * 4, bar);
    };
    int issued = min(L::NST, nch);
    if (lane == 0)
      for (int c = 0; c < issued; ++c) fetch(c);
    __syncthreads();
    for (int c = 0; c < nch; ++c) {
      if (!__syncthreads_and(1)) {      // a copy gave up: wait (bounded) for those in flight
        if (lane == 0)
          for (int i = c; i < issued; ++i) arrived(i);
        break;
      }
      __syncthreads();                  // chunk c's stage is free
      if (c + L::NST < nch) {
        if (lane == 0) fetch(c + L::NST);
        issued = c + L::NST + 1;
      }
    }
    return;
  }
  // st[j] covers key dims dq dk / 4 + 8 j ..; [0], [1]: value column vc, dims 2 t, + 1 of them; [2], [3]: column vc + 8
  float st[KB * 2][4];
  const int vc = 16 * vt + g, d0 = dq * (KB * 16);
#pragma unroll
  for (int j = 0; j < KB * 2; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) st[j][e] = fresh ? 0.f : st_g[(d0 + 8 * j + 2 * t + (e & 1)) * VB + vc + 8 * (e >> 1)];
  // n: lanes 0 .. 3 hold dims d0 + 16 q + 8 vt + 2 t, + 1
  float n[KB][2];
#pragma unroll
  for (int q = 0; q < KB; ++q)
#pragma unroll
    for (int e = 0; e < 2; ++e) n[q][e] = fresh || lane > 3 ? 0.f : st_g[dk * VB + d0 + 16 * q + 8 * vt + 2 * t + e];
  auto put_n = [&](int buf) {              // the limbs' rows
    if (lane < 4) {
#pragma unroll
      for (int q = 0; q < KB; ++q) {
        const int d = d0 + 16 * q + 8 * vt;
        uint8_t* tile = sp + L::OFF_NT + buf * KB * 1024 + (d >> 6) * 1024 + 4 * t;
        uint32_t hi, lo;
        split2(n[q][0], n[q][1], hi, lo);
        *reinterpret_cast<uint32_t*>(tile + piece(0, (d & 63) >> 3)) = hi;
        *reinterpret_cast<uint32_t*>(tile + piece(1, (d & 63) >> 3)) = lo;
      }
    }
  };
  for (int i = tid; i < 2 * KB * 256; i += kScanWork) reinterpret_cast<uint32_t*>(sp + L::OFF_NT)[i] = 0u;
  __syncthreads();
  put_n(0);
  float4* xch = reinterpret_cast<float4*>(sp + L::OFF_X) + lane;          // [warp][row group][2][32]
  // ldmatrix lanes: A rows (row lane & 15, piece half lane >> 4); B rows of two n-tiles (row .., piece half (lane >> 3) & 1)
  const int ar = lane & 15, ah = lane >> 4, br = (lane & 7) + ((lane >> 4) << 3), bh = (lane >> 3) & 1;

  // P of chunk c: 16 rows with this warp's key groups 2 u + ke up to them, and the rows' weights in the state after it
  auto scores = [&](int c) {
    const uint32_t sb = base + stage(c) * L::STAGE, ks = sb + L::OFF_K;
    const float* gt = reinterpret_cast<const float*>(sp + stage(c) * L::STAGE + L::OFF_G);
    const uint32_t ph = base + L::OFF_P + (c & 1) * 2 * L::BLK, pl = ph + L::BLK;
    if (tid < CH) {
      const float b = exp2_fast(gt[tid] - gt[2 * CH - 1]);
      const __nv_bfloat16 hi = __float2bfloat16(b);
      s_b[(c & 1) * CH + tid] = b;
      s_bl[(c & 1) * 2 * CH + tid] = hi;
      s_bl[((c & 1) * 2 + 1) * CH + tid] = __float2bfloat16(b - __bfloat162float(hi));
    }
    float sum[2] = {0.f, 0.f};
    const int tr[2] = {16 * rt + g, 16 * rt + g + 8};
    if (ke <= rt) {
      float x[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) x[j][0] = x[j][1] = x[j][2] = x[j][3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < KB * 4; kk += 2) {
        uint32_t a[2][4];
        const uint32_t blk = (kk >> 2) * L::BLK;
#pragma unroll
        for (int u = 0; u < 2; ++u) ldsm_x4(sb + blk + piece(16 * rt + ar, 2 * ((kk + u) & 3) + ah), a[u]);
#pragma unroll
        for (int u = 0; u < 2; ++u)
          if (2 * u + ke <= rt) {
            uint32_t b[2][4];
#pragma unroll
            for (int w = 0; w < 2; ++w) ldsm_x4(ks + blk + piece(16 * (2 * u + ke) + br, 2 * ((kk + w) & 3) + bh), b[w]);
#pragma unroll
            for (int w = 0; w < 2; ++w) {
              mma_bf16_16816(x[2 * u], a[w][0], a[w][1], a[w][2], a[w][3], b[w][0], b[w][1]);
              mma_bf16_16816(x[2 * u + 1], a[w][0], a[w][1], a[w][2], a[w][3], b[w][2], b[w][3]);
            }
          }
      }
      const float Mt[2] = {gt[CH + tr[0]] - p.q_scale_log2, gt[CH + tr[1]] - p.q_scale_log2};     // the queries' scale rides along
      // all weights before the first store: the stores are barriers for the compiler
#pragma unroll
      for (int u = 0; u < 2; ++u)
        if (2 * u + ke <= rt)
#pragma unroll
          for (int v = 0; v < 2; ++v) {
            const int s0 = 8 * (2 * (2 * u + ke) + v) + 2 * t;
            const float2 as = *reinterpret_cast<const float2*>(gt + s0);
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
              float* e = x[2 * u + v] + 2 * hf;
              e[0] *= exp2_fast(as.x - Mt[hf]);
              e[1] *= exp2_fast(as.y - Mt[hf]);
              if (2 * u + ke == rt) {       // the diagonal: later keys (whose exponent may be above 0) are not seen
                e[0] = s0 <= tr[hf] ? e[0] : 0.f;
                e[1] = s0 + 1 <= tr[hf] ? e[1] : 0.f;
              }
              sum[hf] += e[0] + e[1];
            }
          }
#pragma unroll
      for (int u = 0; u < 2; ++u)
        if (2 * u + ke <= rt)
#pragma unroll
          for (int v = 0; v < 2; ++v)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
              uint32_t hi, lo;
              split2(x[2 * u + v][2 * hf], x[2 * u + v][2 * hf + 1], hi, lo);
              const uint32_t off = piece(tr[hf], 2 * (2 * u + ke) + v) + 4 * t;
              asm volatile("st.shared.u32 [%0], %1;" ::"r"(ph + off), "r"(hi) : "memory");
              asm volatile("st.shared.u32 [%0], %1;" ::"r"(pl + off), "r"(lo) : "memory");
            }
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        sum[hf] += __shfl_xor_sync(0xffffffffu, sum[hf], 1);
        sum[hf] += __shfl_xor_sync(0xffffffffu, sum[hf], 2);
      }
    }
    if (t == 0) {
      s_sum[((c & 1) * 2 + ke) * CH + tr[0]] = sum[0];
      s_sum[((c & 1) * 2 + ke) * CH + tr[1]] = sum[1];
    }
  };

  if (nch > 0) {
    ok = arrived(0);
    if (ok) scores(0);
  }
  float m_last = 0.f;
  for (int c = 0; c < nch; ++c) {
    const uint32_t sb = base + stage(c) * L::STAGE, ks = sb + L::OFF_K, vs = sb + L::OFF_V;
    const float* gt = reinterpret_cast<const float*>(sp + stage(c) * L::STAGE + L::OFF_G);
    const float* bw = s_b + (c & 1) * CH;
    if (!__syncthreads_and(ok)) {      // a copy gave up: leave the state alone
      ok = false;
      break;
    }
    const float m0 = gt[3 * CH], keep = exp2_fast(m0 - gt[2 * CH - 1]);
    m_last = gt[3 * CH - 1];
    // of the rows this warp finishes: the old state's factor, their sum of P and the denominator's floor
    float2 fac[2], psum[2], flr[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = 16 * dq + 8 * u + 2 * t;
      const float2 M = *reinterpret_cast<const float2*>(gt + CH + i), mr = *reinterpret_cast<const float2*>(gt + 2 * CH + i);
      const float2 p0 = *reinterpret_cast<const float2*>(s_sum + (c & 1) * 2 * CH + i);
      const float2 p1 = *reinterpret_cast<const float2*>(s_sum + ((c & 1) * 2 + 1) * CH + i);
      fac[u] = make_float2(exp2_fast(m0 - M.x + p.q_scale_log2), exp2_fast(m0 - M.y + p.q_scale_log2));
      flr[u] = make_float2(exp2_fast(-kLog2e * mr.x), exp2_fast(-kLog2e * mr.y));
      psum[u] = make_float2(p0.x + p1.x, p0.y + p1.y);
    }
    // ---- n . q of 16 rows, half of the dims per warp
    {
      float xn[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int kk = 0; kk < KB * 4; kk += 2)
        if (((kk >> 1) & 1) == ke) {
          uint32_t a[2][4], bn[4];
#pragma unroll
          for (int u = 0; u < 2; ++u) ldsm_x4(sb + (kk >> 2) * L::BLK + piece(16 * rt + ar, 2 * ((kk + u) & 3) + ah), a[u]);
          ldsm_x4(base + L::OFF_NT + (c & 1) * KB * 1024 + (kk >> 2) * 1024 + piece(lane & 7, 2 * (kk & 3) + (lane >> 3)), bn);
          mma_bf16_16816(xn, a[0][0], a[0][1], a[0][2], a[0][3], bn[0], bn[1]);
          mma_bf16_16816(xn, a[1][0], a[1][1], a[1][2], a[1][3], bn[2], bn[3]);
        }
      if (t == 0) {
        s_nq[ke * CH + 16 * rt + g] = xn[0] + xn[1];
        s_nq[ke * CH + 16 * rt + g + 8] = xn[2] + xn[3];
      }
    }
    // ---- O^T [16 value columns][64 rows] from this quarter of the state; rows of the other quarters' warps are handed over
    float o[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < KB; ++kk) {
      uint32_t hi[4], lo[4];
      split2(st[2 * kk][0], st[2 * kk][1], hi[0], lo[0]);
      split2(st[2 * kk][2], st[2 * kk][3], hi[1], lo[1]);
      split2(st[2 * kk + 1][0], st[2 * kk + 1][1], hi[2], lo[2]);
      split2(st[2 * kk + 1][2], st[2 * kk + 1][3], hi[3], lo[3]);
      const int d = d0 + 16 * kk;
      uint32_t b[4][4];
#pragma unroll
      for (int jj = 0; jj < 4; ++jj) ldsm_x4(sb + (d >> 6) * L::BLK + piece(16 * jj + br, ((d & 63) >> 3) + bh), b[jj]);
#pragma unroll
      for (int jj = 0; jj < 4; ++jj)
#pragma unroll
        for (int u = 0; u < 2; ++u) mma_bf16_16816(o[2 * jj + u], hi[0], hi[1], hi[2], hi[3], b[jj][2 * u], b[jj][2 * u + 1]);
#pragma unroll
      for (int jj = 0; jj < 4; ++jj)
#pragma unroll
        for (int u = 0; u < 2; ++u) mma_bf16_16816(o[2 * jj + u], lo[0], lo[1], lo[2], lo[3], b[jj][2 * u], b[jj][2 * u + 1]);
    }
    float4 own[2];
#pragma unroll
    for (int jj = 0; jj < 4; ++jj)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const float4 v = make_float4(o[2 * jj + u][0], o[2 * jj + u][1], o[2 * jj + u][2], o[2 * jj + u][3]);
        if (jj != dq) xch[((warp * 4 + jj) * 2 + u) * 32] = v;
        else own[u] = v;
      }
    uint32_t va[4][4];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) ldsm_x4_trans(vs + piece(16 * kk + br, 4 * (vb & 1) + 2 * vt + bh), va[kk]);
    // ---- the chunk's own values for this warp's 16 rows
    float r[2][4] = {};
    {
      const uint32_t ph = base + L::OFF_P + (c & 1) * 2 * L::BLK, pl = ph + L::BLK;
#pragma unroll
      for (int kk = 0; kk < 4; ++kk)
        if (kk <= dq) {
          uint32_t b[4], bl[4];
          ldsm_x4(ph + piece(16 * dq + br, 2 * kk + bh), b);
          ldsm_x4(pl + piece(16 * dq + br, 2 * kk + bh), bl);
#pragma unroll
          for (int u = 0; u < 2; ++u) mma_bf16_16816(r[u], va[kk][0], va[kk][1], va[kk][2], va[kk][3], b[2 * u], b[2 * u + 1]);
#pragma unroll
          for (int u = 0; u < 2; ++u) mma_bf16_16816(r[u], va[kk][0], va[kk][1], va[kk][2], va[kk][3], bl[2 * u], bl[2 * u + 1]);
        }
    }
    // ---- state after the chunk
#pragma unroll
    for (int j = 0; j < KB * 2; ++j) { st[j][0] *= keep; st[j][1] *= keep; st[j][2] *= keep; st[j][3] *= keep; }
    // n's sums ride along: rows 0 and 1 of one more A tile are the limbs of b
    float ns[KB][4] = {};
    const uint32_t* bl = reinterpret_cast<const uint32_t*>(s_bl + ((c & 1) * 2 + (g & 1)) * CH);
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      const uint32_t b0 = g < 2 ? bl[8 * kk + t] : 0u, b2 = g < 2 ? bl[8 * kk + 4 + t] : 0u;
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 w = *reinterpret_cast<const float2*>(bw + 16 * kk + 8 * (e >> 1) + 2 * t);
        split2(bf16_lo(va[kk][e]) * w.x, bf16_hi(va[kk][e]) * w.y, hi[e], lo[e]);
      }
      uint32_t b[KB][4];
#pragma unroll
      for (int q = 0; q < KB; ++q) {
        const int d = d0 + 16 * q;
        ldsm_x4_trans(ks + (d >> 6) * L::BLK + piece(16 * kk + (lane & 7) + (bh << 3), ((d & 63) >> 3) + ah), b[q]);
      }
#pragma unroll
      for (int q = 0; q < KB; ++q)
#pragma unroll
        for (int u = 0; u < 2; ++u) mma_bf16_16816(st[2 * q + u], hi[0], hi[1], hi[2], hi[3], b[q][2 * u], b[q][2 * u + 1]);
#pragma unroll
      for (int q = 0; q < KB; ++q)
#pragma unroll
        for (int u = 0; u < 2; ++u) mma_bf16_16816(st[2 * q + u], lo[0], lo[1], lo[2], lo[3], b[q][2 * u], b[q][2 * u + 1]);
#pragma unroll
      for (int q = 0; q < KB; ++q) mma_bf16_16816(ns[q], b0, 0u, b2, 0u, vt ? b[q][2] : b[q][0], vt ? b[q][3] : b[q][1]);
    }
#pragma unroll
    for (int q = 0; q < KB; ++q) {
      n[q][0] = fmaf(keep, n[q][0], ns[q][0] + __shfl_down_sync(0xffffffffu, ns[q][0], 4));
      n[q][1] = fmaf(keep, n[q][1], ns[q][1] + __shfl_down_sync(0xffffffffu, ns[q][1], 4));
    }
    put_n((c + 1) & 1);
    if (c + 1 < nch) {
      ok = arrived(c + 1);
      if (ok) scores(c + 1);
    }
    __syncthreads();
    // ---- this warp's 16 rows: the four quarters of the state's part, the denominators
    {
      float* dst = p.o + (size_t)(row0 + c * CH + 16 * dq + 2 * t) * (p.H * p.dv) + h * p.dv + vb * VB + vc;
      const int valid = rows - c * CH - 16 * dq - 2 * t;
      float4 part[2][3];
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int q = 1; q < 4; ++q) part[u][q - 1] = xch[((((dq + q) & 3) * 2 + vt) * 4 + dq) * 64 + u * 32];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int i = 16 * dq + 8 * u + 2 * t;
        const float2 q0 = *reinterpret_cast<const float2*>(s_nq + i), q1 = *reinterpret_cast<const float2*>(s_nq + CH + i);
        const float i0 = __fdividef(1.f, fmaxf(fabsf(fmaf(fac[u].x, q0.x + q1.x, psum[u].x)), flr[u].x) + 1e-6f);
        const float i1 = __fdividef(1.f, fmaxf(fabsf(fmaf(fac[u].y, q0.y + q1.y, psum[u].y)), flr[u].y) + 1e-6f);
        float4 a = own[u];
#pragma unroll
        for (int q = 0; q < 3; ++q) { a.x += part[u][q].x; a.y += part[u][q].y; a.z += part[u][q].z; a.w += part[u][q].w; }
        const float v0 = fmaf(a.x, fac[u].x, r[u][0]) * i0, v1 = fmaf(a.y, fac[u].y, r[u][1]) * i1;
        const float v2 = fmaf(a.z, fac[u].x, r[u][2]) * i0, v3 = fmaf(a.w, fac[u].y, r[u][3]) * i1;
        float* row = dst + (size_t)(8 * u) * (p.H * p.dv);
        if (8 * u < valid) { row[0] = v0; row[8] = v2; }
        if (8 * u + 1 < valid) { row[p.H * p.dv] = v1; row[p.H * p.dv + 8] = v3; }
      }
    }
  }
  if (ok) {
#pragma unroll
    for (int j = 0; j < KB * 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) st_g[(d0 + 8 * j + 2 * t + (e & 1)) * VB + vc + 8 * (e >> 1)] = st[j][e];
    if (lane < 4) {
#pragma unroll
      for (int q = 0; q < KB; ++q)
#pragma unroll
        for (int e = 0; e < 2; ++e) st_g[dk * VB + d0 + 16 * q + 8 * vt + 2 * t + e] = n[q][e];
    }
    if (tid == 0) st_g[state_block(dk) - 4] = m_last;
  }
}

// one warp per (row, head)
__global__ void __launch_bounds__(256) mlstm_out_kernel(const float* __restrict__ o, const __nv_bfloat16* __restrict__ z, int ldz,
                                                        const float* __restrict__ norm, int rows, int H, int dv, int vdim, float eps,
                                                        __nv_bfloat16* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int wid = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int r = wid / H, h = wid - r * H;
  if (r >= rows) return;
  const float* src = o + ((size_t)r * H + h) * dv;
  float ssq = 0.f;
  for (int c = lane * 4; c < dv; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(src + c);
    ssq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float rms = 1.f / sqrtf(warp_sum(ssq) / (float)vdim + eps);
  for (int c = lane * 4; c < dv; c += 128) {
    const float4 v = *reinterpret_cast<const float4*>(src + c);
    const float4 w = *reinterpret_cast<const float4*>(norm + h * dv + c);
    const uint2 zr = *reinterpret_cast<const uint2*>(z + (size_t)r * ldz + h * dv + c);
    auto gate = [](float x) { return 1.f / (1.f + __expf(-x)); };
    *reinterpret_cast<uint2*>(out + ((size_t)r * H + h) * dv + c) =
        make_uint2(pack_bf16(v.x * rms * w.x * gate(bf16_lo(zr.x)), v.y * rms * w.y * gate(bf16_hi(zr.x))),
                   pack_bf16(v.z * rms * w.z * gate(bf16_lo(zr.y)), v.w * rms * w.w * gate(bf16_hi(zr.y))));
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

template <int KB, typename T>
int launch_step(const StepParams& p, cudaStream_t st) {
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
  return (int)cudaLaunchKernelEx(&cfg, mlstm_step_kernel<KB, T>, p);
}

template <typename T>
int launch_step_dk(const StepParams& p, cudaStream_t st) {
  switch (p.dk / 64) {
    case 1: return launch_step<1, T>(p, st);
    case 2: return launch_step<2, T>(p, st);
    case 3: return launch_step<3, T>(p, st);
    case 4: return launch_step<4, T>(p, st);
    case 5: return launch_step<5, T>(p, st);
    case 6: return launch_step<6, T>(p, st);
    case 7: return launch_step<7, T>(p, st);
    case 8: return launch_step<8, T>(p, st);
  }
  return -1;
}

template <int KB>
int launch_scan(const ScanParams& p, int n_segs, cudaStream_t st) {
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(mlstm_scan_kernel<KB>, cudaFuncAttributeMaxDynamicSharedMemorySize, Scan<KB>::SMEM);
    if (e != cudaSuccess) return (int)e;
    configured[dev & 63] = true;
  }
  return b2_launch(mlstm_scan_kernel<KB>, dim3(p.dv / VB, p.H, n_segs), dim3(kScanThreads), Scan<KB>::SMEM, st, true, p);
}

}  // namespace

// fp32 elements of one slot's state
extern "C" int b2_mlstm_state_elems(int H, int dk, int dv) { return H * (dv / VB) * state_block(dk); }

// rows of a sequence are consecutive; part as in StepParams
extern "C" int b2_mlstm_step(const float* part, int slices, int M, int N, int H, int dk, int dv, int dim, int vdim, const int* req,
                             const int* pos, const float* gate_bias, float cap, float eps, const float* norm, float* state,
                             void* out, int f32, void* stream) {
  if (M < 1 || M > 65535 || H < 1 || H > 65535 || slices < 1 || slices > 8 || dk % 64 || dv % 64 || dk > 512 || dv > 512 ||
      N < 2 * H * (dk + dv) + 2 * H || N % 4 || dim < 1 || vdim < 1)
    return -1;
  StepParams p{part, slices, M, N, H, dk, dv, vdim, req, pos, gate_bias, cap, 1.f / sqrtf((float)dim), eps, norm, state, out};
  return f32 ? launch_step_dk<float>(p, (cudaStream_t)stream) : launch_step_dk<__nv_bfloat16>(p, (cudaStream_t)stream);
}

// 1 when the chunked form covers the sizes
extern "C" int b2_mlstm_chunks_ok(int dk, int dv) { return dk % 64 == 0 && dv % 64 == 0 && dk >= 64 && dk <= 256 && dv >= 64 && dv <= 512; }

// Prompt segments.  proj: bf16 [rows][N] q | k | v | g; z: fp32 [rows][ldz] z_i | z_f; segs: n_segs x 4 ints (first row,
// rows, slot, first chunk); gates: fp32 [H][chunks][256]; o: fp32 [rows][H dv]; out bf16 [rows][H dv].
extern "C" int b2_mlstm_segments(const void* proj, int N, const float* z, int ldz, int rows, int H, int dk, int dv, int dim,
                                 int vdim, const int* segs, int n_segs, int chunks, int most_chunks, const int* pos,
                                 const float* gate_bias, float cap, float eps, const float* norm, float* state, float* gates,
                                 float* o, void* out, void* stream) {
  if (rows < 1 || n_segs < 1 || n_segs > 65535 || H > 65535 || !b2_mlstm_chunks_ok(dk, dv) || N != 2 * H * (dk + dv) || ldz < 2 * H ||
      dim < 1 || vdim < 1)
    return -1;
  const size_t gsm = (size_t)most_chunks * 2 * sizeof(float);
  if (gsm > 48 * 1024) return -5;
  cudaStream_t st = (cudaStream_t)stream;
  GatesParams gp{z, ldz, H, dk, dv / VB, chunks, segs, pos, gate_bias, cap, state, gates};
  int rc = b2_launch(mlstm_gates_kernel, dim3(H, n_segs), dim3(256), gsm, st, true, gp);
  if (rc) return rc;
  ScanParams p;
  EncodeTiledFn fn = encode_fn();
  if (!fn) return -100;
  cuuint64_t dims[2] = {(cuuint64_t)N, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)N * 2};
  cuuint32_t box[2] = {64, CH}, estr[2] = {1, 1};
  CUresult r = fn(&p.map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(proj), dims, strides, box, estr,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return -101 - (int)r;
  p.segs = segs; p.pos = pos; p.H = H; p.dv = dv; p.chunks = chunks; p.q_scale_log2 = -0.5f * log2f((float)dim);
  p.gates = gates; p.state = state; p.o = o;
  switch (dk / 64) {
    case 1: rc = launch_scan<1>(p, n_segs, st); break;
    case 2: rc = launch_scan<2>(p, n_segs, st); break;
    case 3: rc = launch_scan<3>(p, n_segs, st); break;
    case 4: rc = launch_scan<4>(p, n_segs, st); break;
  }
  if (rc) return rc;
  return b2_launch(mlstm_out_kernel, dim3((rows * H + 7) / 8), dim3(256), 0, st, true, (const float*)o,
                   (const __nv_bfloat16*)proj + 2 * H * dk + H * dv, N, norm, rows, H, dv, vdim, eps, (__nv_bfloat16*)out);
}

B2_DEFINE_STATUS(mlstm)

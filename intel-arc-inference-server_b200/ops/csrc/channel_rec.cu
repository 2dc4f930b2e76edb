// Recurrences with a matrix state per head and a decay per key channel.  Two update rules share the kernels:
//
//   delta rule     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//                  = S^T q before the write + (k . q) u, so one pass over the state serves both read-outs
//   time mixing    o = S^T q + (sum_d u_d q_d k_d) v;  S <- g S + k v^T
//
//   lowrank_rows_kernel  first halves of low-rank projections as rows for the second ones (bf16 in two limbs, or fp32)
//   delta_prep_kernel    delta rule: short convolution + SiLU of q, k, v, unit q and k, step sizes, decays, output gates
//   wkv_prep_kernel      time mixing: bonus, decays, output gates
//   channel_scan_kernel  the recurrence, rows in order; with few value columns a head's whole read-out stays in one CTA,
//                        which then also norms and gates it
//   channel_out_kernel   head norm and output gate of what the scan left
//
// The prep kernels leave fp32 rows
//   q [Hq dk] | k [Hq dk] | decay [H dk] | v [H dv] | gate [H dv] | s1 [H] | s2 [H]     (both s padded to fours)
// with s1 = beta, s2 = k . q (delta rule) or s1 = bonus (time mixing).  Everything is fp32; models served in 32-bit use the
// same kernels.  A sequence's first row (position 0) starts from zeros whatever its slot holds.
//
// State of one slot: per head and tile of value columns (8, or 4 for more than 256 key dims) the elements in the order in
// which a warp holds them, [dk LK / 4 ... ][32 lanes][4]: lane = (column, dim lane), four key dims each.
#include "common.cuh"

using namespace b2;

namespace {

__device__ __forceinline__ void put4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float dot4(const float4& a, const float4& b) { return a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w; }

// four columns of a projection's row, slices folded in order
__device__ __forceinline__ float4 fold4(const float* p, long long slice, int slices) {
  float4 b[8], a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int s = 0; s < 8; ++s) b[s] = s < slices ? __ldcg(reinterpret_cast<const float4*>(p + s * slice)) : a;
#pragma unroll
  for (int s = 0; s < 8; ++s) { a.x += b[s].x; a.y += b[s].y; a.z += b[s].z; a.w += b[s].w; }
  return a;
}

struct ActLayout {
  int q, k, g, v, z, s1, s2, n;      // first columns, row stride
};
__host__ __device__ inline ActLayout act_layout(int Hq, int H, int dk, int dv) {
  ActLayout a;
  const int h4 = (H + 3) / 4 * 4;
  a.q = 0; a.k = Hq * dk; a.g = 2 * Hq * dk; a.v = a.g + H * dk; a.z = a.v + H * dv; a.s1 = a.z + H * dv; a.s2 = a.s1 + h4;
  a.n = a.s2 + h4;
  return a;
}

// ------------------------------------------------------------------ low-rank projections: rows between the two halves
struct LowRankParams {
  const float* part;       // [slices][M][N]
  int slices, M, N, planes;
  int col[2], rank[2];
  int kp, act;             // columns of a row (fp32) or of one limb; act 1: tanh
  void* out;               // [planes][M][kp] fp32, or bf16 [planes][M][2 kp]: high limbs, low limbs
};

template <typename T>
__global__ void __launch_bounds__(128) lowrank_rows_kernel(const LowRankParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int m = blockIdx.x, pl = blockIdx.y;
  for (int c = threadIdx.x; c < p.kp; c += 128) {
    float v = 0.f;
    if (c < p.rank[pl]) {
      for (int s = 0; s < p.slices; ++s) v += __ldcg(p.part + ((size_t)s * p.M + m) * p.N + p.col[pl] + c);
      if (p.act) v = tanhf(v);
    }
    if constexpr (sizeof(T) == 4) {
      reinterpret_cast<float*>(p.out)[((size_t)pl * p.M + m) * p.kp + c] = v;
    } else {
      __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(p.out) + ((size_t)pl * p.M + m) * 2 * p.kp + c;
      const __nv_bfloat16 hi = __float2bfloat16(v);
      o[0] = hi;
      o[p.kp] = __float2bfloat16(v - __bfloat162float(hi));
    }
  }
}

// Second halves of low-rank projections, either as fp32 slices made by linears, or (in few rows) dots of 32 outputs per
// warp taken here: eight lanes share an output.
struct Second {
  const float* lr;         // [slices][M][n] fp32; null: dots
  int slices, n;
  const void* w;           // [n] rows of ldw elements, the first kp used; element type of the model
  int kp, ldw;
};

// outputs o0 .. o0 + 31 of row m; lane l returns output o0 + l.  x: folded first half, `rank` values at column `col`
template <typename T>
__device__ __forceinline__ float dots32(const Second& s, const float* part, long long slice, int slices, const float* row, int rank,
                                        int o0, bool do_tanh) {
  const int lane = threadIdx.x & 31, sub = lane & 7, grp = lane >> 3;
  float mine = 0.f;
  float acc[8] = {};
  for (int k0 = sub * 8; k0 < s.kp; k0 += 64) {
    float x[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = 0.f;
    for (int q = 0; q < slices; ++q)
#pragma unroll
      for (int e = 0; e < 8; ++e)
        if (k0 + e < rank) x[e] += __ldcg(row + q * slice + k0 + e);
    if (do_tanh) {
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] = tanhf(x[e]);
    }
    if constexpr (sizeof(T) == 2) {
      uint4 w[8];
#pragma unroll
      for (int i = 0; i < 8; ++i)
        w[i] = __ldg(reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(s.w) + (size_t)(o0 + 4 * i + grp) * s.ldw + k0));
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        acc[i] = fmaf(bf16_lo(w[i].x), x[0], acc[i]); acc[i] = fmaf(bf16_hi(w[i].x), x[1], acc[i]);
        acc[i] = fmaf(bf16_lo(w[i].y), x[2], acc[i]); acc[i] = fmaf(bf16_hi(w[i].y), x[3], acc[i]);
        acc[i] = fmaf(bf16_lo(w[i].z), x[4], acc[i]); acc[i] = fmaf(bf16_hi(w[i].z), x[5], acc[i]);
        acc[i] = fmaf(bf16_lo(w[i].w), x[6], acc[i]); acc[i] = fmaf(bf16_hi(w[i].w), x[7], acc[i]);
      }
    } else {
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float4* w = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(s.w) + (size_t)(o0 + 4 * i + grp) * s.ldw + k0);
        const float4 a = w[0], b = w[1];
        acc[i] += a.x * x[0] + a.y * x[1] + a.z * x[2] + a.w * x[3] + b.x * x[4] + b.y * x[5] + b.z * x[6] + b.w * x[7];
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {          // output 4 i + grp
    float v = acc[i];
    v += __shfl_xor_sync(0xffffffffu, v, 1);
    v += __shfl_xor_sync(0xffffffffu, v, 2);
    v += __shfl_xor_sync(0xffffffffu, v, 4);
    const float w = __shfl_sync(0xffffffffu, v, (lane & 3) * 8);
    if ((lane >> 2) == i) mine = w;
  }
  return mine;
}

// ------------------------------------------------------------------ delta rule: what enters the recurrence
struct DeltaPrepParams {
  const float* part;       // [slices][M][N]: q [Hq dk] | k [Hq dk] | v [H dv] | b [H] | a1 | g1 | padding
  int slices, M, N, Hq, H, dk, dv, dim;
  int col_b, col_a1, rank_a1, col_g1, rank_g1;
  const int *req, *pos;
  const float* conv;       // [TP][C], C = 2 Hq dk + H dv; the last row multiplies the row itself
  const float* conv_state; // [slots][TP - 1][C], oldest first
  float* conv_next;        // the same for the sequences of this step
  const float *neg_a, *dt_bias;    // [H] exp(A_log), [H dk]
  Second lr;               // outputs: decay [H dk], gate [H dv] (the latter with their own rows of w)
  float* act;
};

// R rows per warp; tasks of a row: Hq query / key heads, H value heads, blocks of decays, blocks of gates
template <int TP, int R, typename T>
__global__ void __launch_bounds__(128) delta_prep_kernel(const DeltaPrepParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int task = blockIdx.x * 4 + (threadIdx.x >> 5), m0 = blockIdx.y * R, m1 = min(p.M, m0 + R);
  const int C = 2 * p.Hq * p.dk + p.H * p.dv;
  const long long slice = (long long)p.M * p.N;
  const ActLayout L = act_layout(p.Hq, p.H, p.dk, p.dv);
  if (task < p.Hq + p.H) {
    const bool is_v = task >= p.Hq;
    const int head = is_v ? task - p.Hq : task, d = is_v ? p.dv : p.dk, parts = is_v ? 1 : 2;
    const int quads = (d + 127) / 128;
    // a lane's quads one after another; q and k of a head side by side for their product
    for (int m = m0; m < m1; ++m) {
      int before = 0;        // rows of the sequence in this step before row m, up to the taps
#pragma unroll
      for (int j = 1; j < TP; ++j)
        if (before == j - 1 && m - j >= 0 && p.req[m - j] == p.req[m]) before = j;
      const int slot = p.req[m], pos = p.pos[m];
      const bool last = m + 1 == p.M || p.req[m + 1] != slot;
      float ssq[2] = {0.f, 0.f}, kq = 0.f;
      float4 y[2][4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int c = (u * 32 + lane) * 4;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          y[e][u] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (u >= quads || c >= d || e >= parts) continue;
          const int ch = is_v ? 2 * p.Hq * p.dk + head * p.dv + c : e * p.Hq * p.dk + head * p.dk + c;
          float4 win[TP];
#pragma unroll
          for (int j = 0; j < TP; ++j) {      // the input j rows back
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (j <= before) x = fold4(p.part + (size_t)(m - j) * p.N + ch, slice, p.slices);
            else if (pos >= j) x = __ldcg(reinterpret_cast<const float4*>(p.conv_state + ((size_t)slot * (TP - 1) + TP - 1 - (j - before)) * C + ch));
            win[TP - 1 - j] = x;
          }
          float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
          for (int j = 0; j < TP; ++j) {
            const float4 w = __ldg(reinterpret_cast<const float4*>(p.conv + (size_t)j * C + ch));
            a.x = fmaf(w.x, win[j].x, a.x); a.y = fmaf(w.y, win[j].y, a.y); a.z = fmaf(w.z, win[j].z, a.z); a.w = fmaf(w.w, win[j].w, a.w);
          }
          if (last) {
#pragma unroll
            for (int j = 1; j < TP; ++j) put4(p.conv_next + ((size_t)slot * (TP - 1) + j - 1) * C + ch, win[j]);
          }
          a = make_float4(silu_f(a.x), silu_f(a.y), silu_f(a.z), silu_f(a.w));
          y[e][u] = a;
          ssq[e] += dot4(a, a);
        }
        kq += dot4(y[0][u], y[1][u]);
      }
      float* out = p.act + (size_t)m * L.n;
      if (is_v) {
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (u < quads && (u * 32 + lane) * 4 < d) put4(out + L.v + head * p.dv + (u * 32 + lane) * 4, y[0][u]);
        if (lane == 0) {
          float b = 0.f;
          for (int s = 0; s < p.slices; ++s) b += __ldcg(p.part + s * slice + (size_t)m * p.N + p.col_b + head);
          out[L.s1 + head] = sigmoid_f(b);
        }
        continue;
      }
      const float rq = 1.f / sqrtf(warp_sum(ssq[0]) + 1e-6f) / sqrtf((float)p.dim), rk = 1.f / sqrtf(warp_sum(ssq[1]) + 1e-6f);
      kq = warp_sum(kq) * rq * rk;
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int c = (u * 32 + lane) * 4;
        if (u >= quads || c >= d) continue;
        put4(out + L.q + head * p.dk + c, make_float4(y[0][u].x * rq, y[0][u].y * rq, y[0][u].z * rq, y[0][u].w * rq));
        put4(out + L.k + head * p.dk + c, make_float4(y[1][u].x * rk, y[1][u].y * rk, y[1][u].z * rk, y[1][u].w * rk));
      }
      if (lane == 0) out[L.s2 + head] = kq;
    }
    return;
  }
  const int Hk = p.H * p.dk, Hv = p.H * p.dv;
  const int o0 = (task - p.Hq - p.H) * 32;
  if (o0 >= Hk + Hv) return;
  const int o = o0 + lane;
  const bool decay = o0 < Hk;               // whole blocks of 32 are one or the other
  const float nega = decay ? p.neg_a[o / p.dk] : 0.f, bias = decay ? p.dt_bias[o] : 0.f;
  for (int m = m0; m < m1; ++m) {
    float x = 0.f;
    if (p.lr.lr) {
      for (int s = 0; s < p.lr.slices; ++s) x += __ldcg(p.lr.lr + ((size_t)s * p.M + m) * p.lr.n + o);
    } else {
      x = dots32<T>(p.lr, p.part, slice, p.slices, p.part + (size_t)m * p.N + (decay ? p.col_a1 : p.col_g1),
                    decay ? p.rank_a1 : p.rank_g1, o0, false);
    }
    p.act[(size_t)m * L.n + (decay ? L.g + o : L.z + o - Hk)] = decay ? expf(-nega * softplus_f(x + bias)) : sigmoid_f(x);
  }
}

// ------------------------------------------------------------------ time mixing: what enters the recurrence
struct WkvPrepParams {
  const float* part;       // [slices][M][N]: r [H d] | k | v | g | w1 | padding
  int slices, M, N, H, d, rank;
  const float *u, *w0;     // [H d]
  Second lr;               // outputs: decay [H d]
  float* act;
};

template <int R, typename T>
__global__ void __launch_bounds__(128) wkv_prep_kernel(const WkvPrepParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, Hd = p.H * p.d;
  const int task = blockIdx.x * 4 + (threadIdx.x >> 5), m0 = blockIdx.y * R, m1 = min(p.M, m0 + R);
  const long long slice = (long long)p.M * p.N;
  const ActLayout L = act_layout(p.H, p.H, p.d, p.d);
  if (task < p.H) {
    for (int m = m0; m < m1; ++m) {
      const float* row = p.part + (size_t)m * p.N + task * p.d;
      float* out = p.act + (size_t)m * L.n + task * p.d;
      float bonus = 0.f;
      for (int c = lane * 4; c < p.d; c += 128) {
        const float4 r = fold4(row + c, slice, p.slices), k = fold4(row + Hd + c, slice, p.slices);
        const float4 u = *reinterpret_cast<const float4*>(p.u + task * p.d + c);
        bonus += dot4(make_float4(r.x * u.x, r.y * u.y, r.z * u.z, r.w * u.w), k);
        put4(out + L.q + c, r);
        put4(out + L.k + c, k);
        put4(out + L.v + c, fold4(row + 2 * Hd + c, slice, p.slices));
        const float4 g = fold4(row + 3 * Hd + c, slice, p.slices);
        put4(out + L.z + c, make_float4(silu_f(g.x), silu_f(g.y), silu_f(g.z), silu_f(g.w)));
      }
      bonus = warp_sum(bonus);
      if (lane == 0) p.act[(size_t)m * L.n + L.s1 + task] = bonus;
    }
    return;
  }
  const int o0 = (task - p.H) * 32, o = o0 + lane;
  if (o0 >= Hd) return;
  const float w0 = p.w0[o];
  for (int m = m0; m < m1; ++m) {
    float x = 0.f;
    if (p.lr.lr) {
      for (int s = 0; s < p.lr.slices; ++s) x += __ldcg(p.lr.lr + ((size_t)s * p.M + m) * p.lr.n + o);
    } else {
      x = dots32<T>(p.lr, p.part, slice, p.slices, p.part + (size_t)m * p.N + 4 * Hd, p.rank, o0, true);
    }
    p.act[(size_t)m * L.n + L.g + o] = expf(-expf(x + w0));
  }
}

// ------------------------------------------------------------------ the recurrence
typedef unsigned long long f2;
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
  f2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
  f2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f2 both(float v) {
  f2 r;
  asm("mov.b64 %0, {%1, %1};" : "=l"(r) : "f"(v));
  return r;
}
__device__ __forceinline__ float sum2(f2 a) {
  float x, y;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(a));
  return x + y;
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}

struct ScanParams {
  const float* act;
  int Hq, H, dk, dv, vdim;
  const int *req, *pos;
  int M;                   // rows (without `segs`)
  const int* segs;         // [n][4]: first row, rows, slot; null: a sequence per run of equal slots
  float* state;
  const float* conv_next;  // null: no convolution
  float* conv_state;
  int conv_elems;          // of one slot
  float* o;                // [rows][H dv]
  const float* norm;       // fused form: [H dv]
  float eps;
  void* out;               // [rows][H dv]
};

constexpr int kBlockRows = 16;

// ND: key dims per lane, LK: lanes per value column; FUSED: one CTA per head, which finishes its rows
template <int ND, int LK, bool DELTA, bool FUSED, typename T>
__global__ void __launch_bounds__(FUSED ? 512 : 128) channel_scan_kernel(const ScanParams p) {
  constexpr int dk = ND * LK, COLS = 32 / LK;
  extern __shared__ __align__(16) float sm[];
  __shared__ float s_red[2][16];
  const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, dl = lane & (LK - 1), cl = lane / LK;
  const int vb = warps * COLS, h = blockIdx.y, c0 = blockIdx.x * vb, hq = h / (p.H / p.Hq);
  pdl_launch_dependents();
  pdl_wait();
  int row0, rows, slot;
  if (p.segs) {
    row0 = p.segs[blockIdx.z * 4]; rows = p.segs[blockIdx.z * 4 + 1]; slot = p.segs[blockIdx.z * 4 + 2];
  } else {
    row0 = blockIdx.z;
    slot = p.req[row0];
    if (row0 > 0 && p.req[row0 - 1] == slot) return;
    rows = 1;
    while (row0 + rows < p.M && p.req[row0 + rows] == slot) ++rows;
  }
  if (p.conv_next) {        // this step's last inputs become the state
    const int ctas = gridDim.x * gridDim.y, per = (p.conv_elems / 4 + ctas - 1) / ctas;
    const int lo = (blockIdx.y * gridDim.x + blockIdx.x) * per, hi = min(p.conv_elems / 4, lo + per);
    const float4* src = reinterpret_cast<const float4*>(p.conv_next + (size_t)slot * p.conv_elems);
    float4* dst = reinterpret_cast<float4*>(p.conv_state + (size_t)slot * p.conv_elems);
    for (int i = lo + threadIdx.x; i < hi; i += blockDim.x) dst[i] = __ldcg(src + i);
  }
  const ActLayout L = act_layout(p.Hq, p.H, dk, p.dv);
  const int SR = 3 * dk + (FUSED ? 2 : 1) * vb + 4;          // floats of a staged row
  const float* act = p.act + (size_t)row0 * L.n;
  const uint32_t smb = smem_u32(sm);
  auto fetch = [&](int blk) {
    const int r0 = blk * kBlockRows, n = min(kBlockRows, rows - r0);
    const int pieces = 3 * dk / 4 + (FUSED ? 2 : 1) * vb / 4;
    const uint32_t dst = smb + (blk & 1) * kBlockRows * SR * 4;
    for (int i = threadIdx.x; i < n * pieces; i += blockDim.x) {
      const int r = i / pieces, e = (i - r * pieces) * 4;
      int col;
      if (e < dk) col = L.q + hq * dk + e;
      else if (e < 2 * dk) col = L.k + hq * dk + e - dk;
      else if (e < 3 * dk) col = L.g + h * dk + e - 2 * dk;
      else if (!FUSED || e < 3 * dk + vb) col = L.v + h * p.dv + c0 + e - 3 * dk;
      else col = L.z + h * p.dv + e - 3 * dk - vb;
      cp16(dst + (r * SR + e) * 4, act + (size_t)(r0 + r) * L.n + col);
    }
    for (int i = threadIdx.x; i < 2 * n; i += blockDim.x) {
      const float* src = act + (size_t)(r0 + (i >> 1)) * L.n + ((i & 1) ? L.s2 + hq : L.s1 + h);
      asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst + ((i >> 1) * SR + SR - 4 + (i & 1)) * 4), "l"(src) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int blocks = (rows + kBlockRows - 1) / kBlockRows;
  fetch(0);
  // the state: dims (i LK + dl) 4 .. + 3 of column c0 + warp COLS + cl
  float* st = p.state + ((((size_t)slot * p.H + h) * (p.dv / COLS) + c0 / COLS + warp) * (ND / 4)) * 128 + lane * 4;
  f2 S[ND / 2];
  const bool fresh = p.pos[row0] == 0;
#pragma unroll
  for (int i = 0; i < ND / 4; ++i) {
    const ulonglong2 v = fresh ? make_ulonglong2(0ull, 0ull) : __ldcg(reinterpret_cast<const ulonglong2*>(st + i * 128));
    S[2 * i] = v.x;
    S[2 * i + 1] = v.y;
  }
  const int col = warp * COLS + cl;
  const float norm = FUSED ? p.norm[h * p.dv + col] : 0.f;
  for (int b = 0; b < blocks; ++b) {
    if (b + 1 < blocks) {
      fetch(b + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int n = min(kBlockRows, rows - b * kBlockRows);
    const float* base = sm + (b & 1) * kBlockRows * SR;
    for (int r = 0; r < n; ++r) {
      const float* row = base + r * SR;
      const ulonglong2* q = reinterpret_cast<const ulonglong2*>(row) + dl;
      const ulonglong2* k = reinterpret_cast<const ulonglong2*>(row + dk) + dl;
      const ulonglong2* g = reinterpret_cast<const ulonglong2*>(row + 2 * dk) + dl;
      const float v = row[3 * dk + col];
      const float2 s12 = *reinterpret_cast<const float2*>(row + SR - 4);
      float o;
      if constexpr (DELTA) {
        f2 pq[2] = {0ull, 0ull}, pk[2] = {0ull, 0ull}, kk[ND / 2];
#pragma unroll
        for (int i = 0; i < ND / 4; ++i) {
          const ulonglong2 gv = g[i * LK], kv = k[i * LK], qv = q[i * LK];
          kk[2 * i] = kv.x;
          kk[2 * i + 1] = kv.y;
          S[2 * i] = mul2(S[2 * i], gv.x);
          S[2 * i + 1] = mul2(S[2 * i + 1], gv.y);
          pk[0] = fma2(S[2 * i], kv.x, pk[0]);
          pk[1] = fma2(S[2 * i + 1], kv.y, pk[1]);
          pq[0] = fma2(S[2 * i], qv.x, pq[0]);
          pq[1] = fma2(S[2 * i + 1], qv.y, pq[1]);
        }
        float a = sum2(pk[0]) + sum2(pk[1]);
        o = sum2(pq[0]) + sum2(pq[1]);
#pragma unroll
        for (int x = 1; x < LK; x <<= 1) {
          a += __shfl_xor_sync(0xffffffffu, a, x);
          o += __shfl_xor_sync(0xffffffffu, o, x);
        }
        const float u = s12.x * (v - a);
        const f2 u2 = both(u);
#pragma unroll
        for (int i = 0; i < ND / 2; ++i) S[i] = fma2(kk[i], u2, S[i]);
        o = fmaf(s12.y, u, o);
      } else {
        f2 pq[2] = {0ull, 0ull};
        const f2 v2 = both(v);
#pragma unroll
        for (int i = 0; i < ND / 4; ++i) {
          const ulonglong2 gv = g[i * LK], kv = k[i * LK], qv = q[i * LK];
          pq[0] = fma2(S[2 * i], qv.x, pq[0]);
          pq[1] = fma2(S[2 * i + 1], qv.y, pq[1]);
          S[2 * i] = fma2(kv.x, v2, mul2(S[2 * i], gv.x));
          S[2 * i + 1] = fma2(kv.y, v2, mul2(S[2 * i + 1], gv.y));
        }
        o = sum2(pq[0]) + sum2(pq[1]);
#pragma unroll
        for (int x = 1; x < LK; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
        o = fmaf(s12.x, v, o);
      }
      const size_t at = (size_t)(row0 + b * kBlockRows + r) * (p.H * p.dv) + h * p.dv + c0 + col;
      if constexpr (FUSED) {
        float ssq = o * o;
#pragma unroll
        for (int x = LK; x < 32; x <<= 1) ssq += __shfl_xor_sync(0xffffffffu, ssq, x);
        if (lane == 0) s_red[r & 1][warp] = ssq;
        __syncthreads();
        float tot = 0.f;
        for (int w = 0; w < warps; ++w) tot += s_red[r & 1][w];
        if (dl == 0) put(reinterpret_cast<T*>(p.out) + at, o / sqrtf(tot / (float)p.vdim + p.eps) * norm * row[3 * dk + vb + col]);
      } else {
        if (dl == 0) p.o[at] = o;
      }
    }
    __syncthreads();       // the block's rows are read: the next fetch may overwrite them
  }
#pragma unroll
  for (int i = 0; i < ND / 4; ++i) *reinterpret_cast<ulonglong2*>(st + i * 128) = make_ulonglong2(S[2 * i], S[2 * i + 1]);
}

// one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(256) channel_out_kernel(const float* __restrict__ o, const float* __restrict__ act, int ldact, int col_z,
                                                          const float* __restrict__ norm, int rows, int H, int dv, int vdim, float eps,
                                                          T* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const int wid = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int r = wid / H, h = wid - r * H;
  if (r >= rows) return;
  const float* src = o + ((size_t)r * H + h) * dv;
  float ssq = 0.f;
  for (int c = lane * 4; c < dv; c += 128) {
    const float4 v = __ldcg(reinterpret_cast<const float4*>(src + c));
    ssq += dot4(v, v);
  }
  const float rms = 1.f / sqrtf(warp_sum(ssq) / (float)vdim + eps);
  for (int c = lane * 4; c < dv; c += 128) {
    const float4 v = __ldcg(reinterpret_cast<const float4*>(src + c));
    const float4 w = *reinterpret_cast<const float4*>(norm + h * dv + c);
    const float4 z = __ldcg(reinterpret_cast<const float4*>(act + (size_t)r * ldact + col_z + h * dv + c));
    put4(out + ((size_t)r * H + h) * dv + c, make_float4(v.x * rms * w.x * z.x, v.y * rms * w.y * z.y, v.z * rms * w.z * z.z, v.w * rms * w.w * z.w));
  }
}

// key dims of the kernels: 64, 128, 192, 256 with four lanes per column, 384 and 512 with eight
bool dk_ok(int dk) { return dk == 64 || dk == 128 || dk == 192 || dk == 256 || dk == 384 || dk == 512; }

template <int ND, int LK, bool DELTA, bool FUSED, typename T>
int launch_scan(const ScanParams& p, int seqs, cudaStream_t st) {
  constexpr int COLS = 32 / LK;
  const int warps = FUSED ? p.dv / COLS : 4, vb = warps * COLS;
  const int smem = 2 * kBlockRows * (3 * ND * LK + (FUSED ? 2 : 1) * vb + 4) * 4;
  if (smem > 227 * 1024 - 1024) return -6;
  if (smem > 48 * 1024) {
    static int configured[64] = {};
    int dev = 0;
    cudaGetDevice(&dev);
    if (configured[dev & 63] < smem) {
      cudaError_t e = cudaFuncSetAttribute(channel_scan_kernel<ND, LK, DELTA, FUSED, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
      if (e != cudaSuccess) return (int)e;
      configured[dev & 63] = smem;
    }
  }
  return b2_launch(channel_scan_kernel<ND, LK, DELTA, FUSED, T>, dim3(p.dv / vb, p.H, seqs), dim3(warps * 32), smem, st, true, p);
}

template <bool DELTA, bool FUSED, typename T>
int launch_scan_dk(const ScanParams& p, int seqs, cudaStream_t st) {
  switch (p.dk) {
    case 64: return launch_scan<16, 4, DELTA, FUSED, T>(p, seqs, st);
    case 128: return launch_scan<32, 4, DELTA, FUSED, T>(p, seqs, st);
    case 192: return launch_scan<48, 4, DELTA, FUSED, T>(p, seqs, st);
    case 256: return launch_scan<64, 4, DELTA, FUSED, T>(p, seqs, st);
    case 384: return FUSED ? -1 : launch_scan<48, 8, DELTA, false, T>(p, seqs, st);
    case 512: return FUSED ? -1 : launch_scan<64, 8, DELTA, false, T>(p, seqs, st);
  }
  return -1;
}

template <int TP, typename T>
int launch_delta_prep(const DeltaPrepParams& p, int tasks, cudaStream_t st) {
  if (p.M > 64) return b2_launch(delta_prep_kernel<TP, 4, T>, dim3((tasks + 3) / 4, (p.M + 3) / 4), dim3(128), 0, st, true, p);
  return b2_launch(delta_prep_kernel<TP, 1, T>, dim3((tasks + 3) / 4, p.M), dim3(128), 0, st, true, p);
}

template <typename T>
int delta_prep_taps(const DeltaPrepParams& p, int taps, int tasks, cudaStream_t st) {
  switch (taps) {
    case 4: return launch_delta_prep<4, T>(p, tasks, st);
    case 8: return launch_delta_prep<8, T>(p, tasks, st);
    case 16: return launch_delta_prep<16, T>(p, tasks, st);
  }
  return -1;
}

}  // namespace

// columns of a prepared row
extern "C" int b2_channel_act_cols(int Hq, int H, int dk, int dv) { return act_layout(Hq, H, dk, dv).n; }

// part: fp32 [slices][M][N]; planes (up to 2) of `rank` columns at `col`; out: see LowRankParams
extern "C" int b2_lowrank_rows(const float* part, int slices, int M, int N, int planes, int col0, int rank0, int col1, int rank1, int kp,
                               int act, void* out, int f32, void* stream) {
  if (M < 1 || slices < 1 || planes < 1 || planes > 2 || rank0 > kp || rank1 > kp) return -1;
  LowRankParams p{part, slices, M, N, planes, {col0, col1}, {rank0, rank1}, kp, act, out};
  return f32 ? b2_launch(lowrank_rows_kernel<float>, dim3(M, planes), dim3(128), 0, (cudaStream_t)stream, true, p)
             : b2_launch(lowrank_rows_kernel<__nv_bfloat16>, dim3(M, planes), dim3(128), 0, (cudaStream_t)stream, true, p);
}

// taps: 4, 8 or 16 (shorter convolutions padded with zeros at the old end).  lr: fp32 [lr_slices][M][H (dk + dv)], or null
// with w2 [H (dk + dv)] rows of ldw elements (kp used) in the model's element type, which read a1 (decays) and g1 (gates).
extern "C" int b2_delta_prep(const float* part, int slices, int M, int N, int Hq, int H, int dk, int dv, int dim, int col_b, int col_a1,
                             int rank_a1, int col_g1, int rank_g1, const int* req, const int* pos, int taps, const float* conv,
                             const float* conv_state, float* conv_next, const float* neg_a, const float* dt_bias, const float* lr,
                             int lr_slices, const void* w2, int kp, int ldw, float* act, int f32, void* stream) {
  if (M < 1 || slices < 1 || slices > 8 || Hq < 1 || H % Hq || !dk_ok(dk) || dv % 64 || dv < 64 || dv > 512 || N % 4 || kp % 64 ||
      rank_a1 > kp || rank_g1 > kp || ldw < kp || ldw % 8 || (!lr && !w2))
    return -1;
  DeltaPrepParams p{part, slices, M, N, Hq, H, dk, dv, dim, col_b, col_a1, rank_a1, col_g1, rank_g1, req, pos, conv, conv_state,
                    conv_next, neg_a, dt_bias, {lr, lr_slices, H * (dk + dv), w2, kp, ldw}, act};
  const int tasks = Hq + H + H * (dk + dv) / 32;
  return f32 ? delta_prep_taps<float>(p, taps, tasks, (cudaStream_t)stream) : delta_prep_taps<__nv_bfloat16>(p, taps, tasks, (cudaStream_t)stream);
}

// part: r | k | v | g (H d columns each) | w1; lr: fp32 [lr_slices][M][H d], or null with w2 as above, [H d] rows
extern "C" int b2_wkv_prep(const float* part, int slices, int M, int N, int H, int d, int rank, const float* u, const float* w0,
                           const float* lr, int lr_slices, const void* w2, int kp, int ldw, float* act, int f32, void* stream) {
  if (M < 1 || slices < 1 || slices > 8 || H < 1 || !dk_ok(d) || N % 4 || kp % 64 || rank > kp || ldw < kp || ldw % 8 ||
      (!lr && !w2))
    return -1;
  WkvPrepParams p{part, slices, M, N, H, d, rank, u, w0, {lr, lr_slices, H * d, w2, kp, ldw}, act};
  const int tasks = (H + H * d / 32 + 3) / 4;
  cudaStream_t st = (cudaStream_t)stream;
  if (M > 64)
    return f32 ? b2_launch(wkv_prep_kernel<4, float>, dim3(tasks, (M + 3) / 4), dim3(128), 0, st, true, p)
               : b2_launch(wkv_prep_kernel<4, __nv_bfloat16>, dim3(tasks, (M + 3) / 4), dim3(128), 0, st, true, p);
  return f32 ? b2_launch(wkv_prep_kernel<1, float>, dim3(tasks, M), dim3(128), 0, st, true, p)
             : b2_launch(wkv_prep_kernel<1, __nv_bfloat16>, dim3(tasks, M), dim3(128), 0, st, true, p);
}

// fp32 elements of one slot's state
extern "C" int b2_channel_state_elems(int H, int dk, int dv) { return H * dk * dv; }

// 1 when the scan's CTA holds a whole head and writes the finished rows itself
extern "C" int b2_channel_fused(int dk, int dv) { return dk <= 256 && dv <= 128; }

// The recurrence over prepared rows.  segs null: rows 0 .. M - 1, a sequence per run of equal `req`; else n_segs x 4 ints
// (first row, rows, slot, unused).  out [rows][H dv]; raw: fp32 of the same shape, unused where b2_channel_fused says so and
// segs is null.  delta 1: delta rule, 0: time mixing.
extern "C" int b2_channel_scan(const float* act, int delta, int M, int Hq, int H, int dk, int dv, int vdim, const int* req, const int* pos,
                               const int* segs, int n_segs, float* state, const float* conv_next, float* conv_state, int conv_elems,
                               const float* norm, float eps, float* raw, void* out, int f32, void* stream) {
  if (M < 1 || H < 1 || H > 65535 || Hq < 1 || H % Hq || !dk_ok(dk) || dv % 64 || dv < 64 || dv > 512 || conv_elems % 4) return -1;
  const int seqs = segs ? n_segs : M;
  if (seqs < 1 || seqs > 65535) return -2;
  ScanParams p{act, Hq, H, dk, dv, vdim, req, pos, M, segs, state, conv_next, conv_state, conv_elems, raw, norm, eps, out};
  cudaStream_t st = (cudaStream_t)stream;
  if (!segs && b2_channel_fused(dk, dv)) {
    if (delta) return f32 ? launch_scan_dk<true, true, float>(p, seqs, st) : launch_scan_dk<true, true, __nv_bfloat16>(p, seqs, st);
    return f32 ? launch_scan_dk<false, true, float>(p, seqs, st) : launch_scan_dk<false, true, __nv_bfloat16>(p, seqs, st);
  }
  if (!raw) return -3;
  const int rc = delta ? launch_scan_dk<true, false, float>(p, seqs, st) : launch_scan_dk<false, false, float>(p, seqs, st);
  if (rc) return rc;
  const ActLayout L = act_layout(Hq, H, dk, dv);
  const dim3 grid((unsigned)(((long long)M * H + 7) / 8));
  return f32 ? b2_launch(channel_out_kernel<float>, grid, dim3(256), 0, st, true, (const float*)raw, act, L.n, L.z, norm, M, H, dv, vdim, eps, (float*)out)
             : b2_launch(channel_out_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, true, (const float*)raw, act, L.n, L.z, norm, M, H, dv, vdim, eps, (__nv_bfloat16*)out);
}

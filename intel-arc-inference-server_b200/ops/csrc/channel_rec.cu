// Recurrences with a matrix state per head and a decay per key channel.  Two update rules share the kernels:
//
//   delta rule     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//                  = S^T q before the write + (k . q) u, so one pass over the state serves both read-outs
//   time mixing    o = S^T q + (sum_d u_d q_d k_d) v;  S <- g S + k v^T
//
//   lowrank_rows_kernel  first halves of low-rank projections as rows for the second ones (bf16 in two limbs, or fp32)
//   delta_prep_kernel    delta rule: short convolution + SiLU of q, k, v, unit q and k, step sizes, decays, output gates
//   wkv_prep_kernel      time mixing: bonus, decays, output gates
//   channel_rows_kernel  the recurrence, rows one by one; with few value columns a head's whole read-out stays in one CTA, which
//                        then also norms and gates it
//   channel_groups_kernel  the recurrence over prompt segments, four rows at a time
//   channel_out_kernel   head norm and output gate of what the scan left
//
// The prep kernels leave fp32 rows
//   q [Hq dk] | k [Hq dk] | decay [H dk] | v [H dv] | gate [H dv] | s1 [H] | s2 [H]     (both s padded to fours)
// with s1 = beta, s2 = k . q (delta rule) or s1 = bonus (time mixing).  Everything is fp32; models served in 32-bit use the
// same kernels.  A sequence's first row (position 0) starts from zeros whatever its slot holds.
//
// State of one slot: per head and tile of value columns (8, or 4 for more than 256 key dims) the elements in the order in
// which a warp holds them: [dk / 32][columns per lane][32 lanes][4 key dims].
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
  if (slices == 1) return __ldcg(reinterpret_cast<const float4*>(p));
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

// second half of a low-rank projection from its fp32 slices: four outputs of R rows
template <int R>
__device__ __forceinline__ void second4(const Second& s, int M, int m0, int m1, int o, float4 (&x)[R]) {
#pragma unroll
  for (int r = 0; r < R; ++r)
    if (m0 + r < m1) x[r] = fold4(s.lr + (size_t)(m0 + r) * s.n + o, (long long)M * s.n, s.slices);
}

// R rows per warp, QN quads of a head's columns per lane.  Tasks of a row: Hq query / key heads, H value heads, then decays and
// gates, 32 outputs (dots) or 128 (slices) each
template <int TP, int R, int QN, typename T>
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
    int before[R];           // rows of the sequence in this step before the row, up to the taps
    bool last[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      before[r] = 0;
      last[r] = false;
      const int m = m0 + r;
      if (m >= m1) continue;
#pragma unroll
      for (int j = 1; j < TP; ++j)
        if (before[r] == j - 1 && m - j >= 0 && p.req[m - j] == p.req[m]) before[r] = j;
      last[r] = m + 1 == p.M || p.req[m + 1] != p.req[m];
    }
    float4 y[R][2][QN];
#pragma unroll
    for (int u = 0; u < QN; ++u) {
      const int c = (u * 32 + lane) * 4;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
#pragma unroll
        for (int r = 0; r < R; ++r) y[r][e][u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c >= d || e >= parts) continue;
        const int ch = is_v ? 2 * p.Hq * p.dk + head * p.dv + c : e * p.Hq * p.dk + head * p.dk + c;
        float4 xs[R + TP - 1];
#pragma unroll
        for (int i = 0; i < R + TP - 1; ++i) {
          const int m = m0 - (TP - 1) + i;
          xs[i] = m >= 0 && m < m1 ? fold4(p.part + (size_t)m * p.N + ch, slice, p.slices) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        float4 w[TP];
#pragma unroll
        for (int j = 0; j < TP; ++j) w[j] = __ldg(reinterpret_cast<const float4*>(p.conv + (size_t)j * C + ch));
#pragma unroll
        for (int r = 0; r < R; ++r) {
          const int m = m0 + r;
          if (m >= m1) continue;
          float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
          if (before[r] == TP - 1 && !last[r]) {
#pragma unroll
            for (int j = 0; j < TP; ++j) {
              const float4 x = xs[r + j];
              a.x = fmaf(w[j].x, x.x, a.x); a.y = fmaf(w[j].y, x.y, a.y); a.z = fmaf(w[j].z, x.z, a.z); a.w = fmaf(w[j].w, x.w, a.w);
            }
          } else {
            const int slot = p.req[m], pos = p.pos[m];
#pragma unroll
            for (int j = 0; j < TP; ++j) {       // the input TP - 1 - j rows back: of this step, of the state, or none
              const int back = TP - 1 - j;
              float4 x = xs[r + j];
              if (back > before[r])
                x = pos >= back ? __ldcg(reinterpret_cast<const float4*>(p.conv_state + ((size_t)slot * (TP - 1) + j + before[r]) * C + ch))
                                : make_float4(0.f, 0.f, 0.f, 0.f);
              a.x = fmaf(w[j].x, x.x, a.x); a.y = fmaf(w[j].y, x.y, a.y); a.z = fmaf(w[j].z, x.z, a.z); a.w = fmaf(w[j].w, x.w, a.w);
              if (last[r] && j > 0) put4(p.conv_next + ((size_t)slot * (TP - 1) + j - 1) * C + ch, x);
            }
          }
          y[r][e][u] = make_float4(silu_f(a.x), silu_f(a.y), silu_f(a.z), silu_f(a.w));
        }
      }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int m = m0 + r;
      if (m >= m1) continue;
      float* out = p.act + (size_t)m * L.n;
      if (is_v) {
#pragma unroll
        for (int u = 0; u < QN; ++u)
          if ((u * 32 + lane) * 4 < d) put4(out + L.v + head * p.dv + (u * 32 + lane) * 4, y[r][0][u]);
        if (lane == 0) {
          float b = 0.f;
          for (int s = 0; s < p.slices; ++s) b += __ldcg(p.part + s * slice + (size_t)m * p.N + p.col_b + head);
          out[L.s1 + head] = sigmoid_f(b);
        }
        continue;
      }
      float sq = 0.f, sk = 0.f, kq = 0.f;
#pragma unroll
      for (int u = 0; u < QN; ++u) {
        sq += dot4(y[r][0][u], y[r][0][u]);
        sk += dot4(y[r][1][u], y[r][1][u]);
        kq += dot4(y[r][0][u], y[r][1][u]);
      }
      const float rq = 1.f / sqrtf((warp_sum(sq) + 1e-6f) * (float)p.dim), rk = 1.f / sqrtf(warp_sum(sk) + 1e-6f);
      kq = warp_sum(kq) * rq * rk;
#pragma unroll
      for (int u = 0; u < QN; ++u) {
        const int c = (u * 32 + lane) * 4;
        if (c >= d) continue;
        const float4 a = y[r][0][u], b = y[r][1][u];
        put4(out + L.q + head * p.dk + c, make_float4(a.x * rq, a.y * rq, a.z * rq, a.w * rq));
        put4(out + L.k + head * p.dk + c, make_float4(b.x * rk, b.y * rk, b.z * rk, b.w * rk));
      }
      if (lane == 0) out[L.s2 + head] = kq;
    }
    return;
  }
  const int Hk = p.H * p.dk, Hv = p.H * p.dv;
  if (p.lr.lr) {
    const int o = ((task - p.Hq - p.H) * 32 + lane) * 4;
    if (o >= Hk + Hv) return;
    const bool decay = o < Hk;
    float4 x[R];
    second4<R>(p.lr, p.M, m0, m1, o, x);
    const float nega = decay ? p.neg_a[o / p.dk] : 0.f;
    const float4 b = decay ? *reinterpret_cast<const float4*>(p.dt_bias + o) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      if (m0 + r >= m1) continue;
      auto f = [&](float v, float bias) { return decay ? expf(-nega * softplus_f(v + bias)) : sigmoid_f(v); };
      put4(p.act + (size_t)(m0 + r) * L.n + (decay ? L.g + o : L.z + o - Hk), make_float4(f(x[r].x, b.x), f(x[r].y, b.y), f(x[r].z, b.z), f(x[r].w, b.w)));
    }
    return;
  }
  const int o0 = (task - p.Hq - p.H) * 32, o = o0 + lane;
  if (o0 >= Hk + Hv) return;
  const bool decay = o0 < Hk;               // whole blocks of 32 are one or the other
  const float nega = decay ? p.neg_a[o / p.dk] : 0.f, bias = decay ? p.dt_bias[o] : 0.f;
  for (int m = m0; m < m1; ++m) {
    const float x = dots32<T>(p.lr, p.part, slice, p.slices, p.part + (size_t)m * p.N + (decay ? p.col_a1 : p.col_g1),
                              decay ? p.rank_a1 : p.rank_g1, o0, false);
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

// R rows per warp; tasks of a row: H heads, then decays, 32 outputs (dots) or 128 (slices) each
template <int R, typename T>
__global__ void __launch_bounds__(128) wkv_prep_kernel(const WkvPrepParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, Hd = p.H * p.d;
  const int task = blockIdx.x * 4 + (threadIdx.x >> 5), m0 = blockIdx.y * R, m1 = min(p.M, m0 + R);
  const long long slice = (long long)p.M * p.N;
  const ActLayout L = act_layout(p.H, p.H, p.d, p.d);
  if (task < p.H) {
    float bonus[R];
#pragma unroll
    for (int r = 0; r < R; ++r) bonus[r] = 0.f;
    for (int c = lane * 4; c < p.d; c += 128) {
      const int col = task * p.d + c;
      float4 x[R][4];
#pragma unroll
      for (int r = 0; r < R; ++r)
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (m0 + r < m1) x[r][i] = fold4(p.part + (size_t)(m0 + r) * p.N + i * Hd + col, slice, p.slices);
      const float4 u = *reinterpret_cast<const float4*>(p.u + col);
#pragma unroll
      for (int r = 0; r < R; ++r) {
        if (m0 + r >= m1) continue;
        float* out = p.act + (size_t)(m0 + r) * L.n + col;
        const float4 a = x[r][0], g = x[r][3];
        bonus[r] += dot4(make_float4(a.x * u.x, a.y * u.y, a.z * u.z, a.w * u.w), x[r][1]);
        put4(out + L.q, a);
        put4(out + L.k, x[r][1]);
        put4(out + L.v, x[r][2]);
        put4(out + L.z, make_float4(silu_f(g.x), silu_f(g.y), silu_f(g.z), silu_f(g.w)));
      }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const float b = warp_sum(bonus[r]);
      if (lane == 0 && m0 + r < m1) p.act[(size_t)(m0 + r) * L.n + L.s1 + task] = b;
    }
    return;
  }
  if (p.lr.lr) {
    const int o = ((task - p.H) * 32 + lane) * 4;
    if (o >= Hd) return;
    float4 x[R];
    second4<R>(p.lr, p.M, m0, m1, o, x);
    const float4 b = *reinterpret_cast<const float4*>(p.w0 + o);
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (m0 + r < m1)
        put4(p.act + (size_t)(m0 + r) * L.n + L.g + o, make_float4(expf(-expf(x[r].x + b.x)), expf(-expf(x[r].y + b.y)),
                                                                    expf(-expf(x[r].z + b.z)), expf(-expf(x[r].w + b.w))));
    return;
  }
  const int o0 = (task - p.H) * 32, o = o0 + lane;
  if (o0 >= Hd) return;
  const float w0 = p.w0[o];
  for (int m = m0; m < m1; ++m) {
    const float x = dots32<T>(p.lr, p.part, slice, p.slices, p.part + (size_t)m * p.N + 4 * Hd, p.rank, o0, true);
    p.act[(size_t)m * L.n + L.g + o] = expf(-expf(x + w0));
  }
}

// ------------------------------------------------------------------ the recurrence
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

constexpr int kBlockRows = 16;     // rows staged at a time
constexpr int kGroup = 4;          // rows of a group in the scan of segments

// A warp holds the state of 4 NC value columns: lane = (dim lane dl = lane / 4, cl = lane % 4), columns cl NC + j of its tile, key
// dims (8 i + dl) 4 .. + 3.  The dim lanes are the upper lane bits: the four lanes that read the same 16 bytes of a shared row
// are then neighbours, which halves the wavefronts of the load.
template <int ND, int NC>
__device__ __forceinline__ void load_state(float4 (&S)[ND / 4][NC], const float* st, bool fresh) {
#pragma unroll
  for (int i = 0; i < ND / 4; ++i)
#pragma unroll
    for (int j = 0; j < NC; ++j)
      S[i][j] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : __ldcg(reinterpret_cast<const float4*>(st + (i * NC + j) * 128));
}
template <int ND, int NC>
__device__ __forceinline__ void store_state(const float4 (&S)[ND / 4][NC], float* st) {
#pragma unroll
  for (int i = 0; i < ND / 4; ++i)
#pragma unroll
    for (int j = 0; j < NC; ++j) *reinterpret_cast<float4*>(st + (i * NC + j) * 128) = S[i][j];
}
__device__ __forceinline__ float fdot4(const float4& a, const float4& b, float c) {
  return fmaf(a.w, b.w, fmaf(a.z, b.z, fmaf(a.y, b.y, fmaf(a.x, b.x, c))));
}
__device__ __forceinline__ float4 mul4(const float4& a, const float4& b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float4 axpy4(float a, const float4& x, const float4& y) {
  return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}

// which sequence a CTA walks; false: none
__device__ __forceinline__ bool find_rows(const ScanParams& p, int& row0, int& rows, int& slot) {
  if (p.segs) {
    row0 = p.segs[blockIdx.z * 4]; rows = p.segs[blockIdx.z * 4 + 1]; slot = p.segs[blockIdx.z * 4 + 2];
    return true;
  }
  row0 = blockIdx.z;
  slot = p.req[row0];
  if (row0 > 0 && p.req[row0 - 1] == slot) return false;
  rows = 1;
  while (row0 + rows < p.M && p.req[row0 + rows] == slot) ++rows;
  return true;
}

// this step's last convolution inputs become the sequence's state
__device__ __forceinline__ void commit_inputs(const ScanParams& p, int slot) {
  if (!p.conv_next) return;
  const int ctas = gridDim.x * gridDim.y, per = (p.conv_elems / 4 + ctas - 1) / ctas;
  const int lo = (blockIdx.y * gridDim.x + blockIdx.x) * per, hi = min(p.conv_elems / 4, lo + per);
  const float4* src = reinterpret_cast<const float4*>(p.conv_next + (size_t)slot * p.conv_elems);
  float4* dst = reinterpret_cast<float4*>(p.conv_state + (size_t)slot * p.conv_elems);
  for (int i = lo + threadIdx.x; i < hi; i += blockDim.x) dst[i] = __ldcg(src + i);
}

// A CTA's share of staged rows: q | k | decay | v of its columns | (gates of its columns) | s1, s2, padding
template <int dk, bool GATES>
struct Stage {
  int vb, SR;
  __device__ Stage(int cols) : vb(cols), SR(3 * dk + (GATES ? 2 : 1) * cols + 4) {}
  // rows r0 .. r0 + n - 1 of the sequence whose first row is at `act`
  __device__ void fetch(uint32_t dst, const ScanParams& p, const ActLayout& L, const float* act, int r0, int n, int h, int hq, int c0) const {
    const int pieces = 3 * dk / 4 + (GATES ? 2 : 1) * vb / 4;
    for (int e4 = threadIdx.x; e4 < pieces; e4 += blockDim.x) {
      const int e = e4 * 4;
      int col;
      if (e < dk) col = L.q + hq * dk + e;
      else if (e < 2 * dk) col = L.k + hq * dk + e - dk;
      else if (e < 3 * dk) col = L.g + h * dk + e - 2 * dk;
      else if (!GATES || e < 3 * dk + vb) col = L.v + h * p.dv + c0 + e - 3 * dk;
      else col = L.z + h * p.dv + c0 + e - 3 * dk - vb;
      const float* src = act + (size_t)r0 * L.n + col;
      uint32_t d = dst + e * 4;
      for (int r = 0; r < n; ++r, src += L.n, d += SR * 4) cp16(d, src);
    }
    for (int i = threadIdx.x; i < 2 * n; i += blockDim.x) {
      const float* src = act + (size_t)(r0 + (i >> 1)) * L.n + ((i & 1) ? L.s2 + hq : L.s1 + h);
      asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst + ((i >> 1) * SR + SR - 4 + (i & 1)) * 4), "l"(src) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
};

// Rows of a step one after another.  ND: key dims per lane, NC: value columns per lane; FUSED: one CTA per head, which
// finishes its rows.
template <int ND, int NC, bool DELTA, bool FUSED, typename T>
__global__ void __launch_bounds__(FUSED ? 512 : 128) channel_rows_kernel(const ScanParams p) {
  constexpr int LK = 8, CL = 4, dk = ND * LK, COLS = CL * NC;
  extern __shared__ __align__(16) float sm[];
  __shared__ float s_red[2][32];
  const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, dl = lane / CL, cl = lane % CL;
  const int vb = warps * COLS, h = blockIdx.y, c0 = blockIdx.x * vb, hq = h / (p.H / p.Hq);
  pdl_launch_dependents();
  pdl_wait();
  int row0, rows, slot;
  if (!find_rows(p, row0, rows, slot)) return;
  commit_inputs(p, slot);
  const ActLayout L = act_layout(p.Hq, p.H, dk, p.dv);
  const Stage<dk, FUSED> stage(vb);
  const int SR = stage.SR;
  const float* act = p.act + (size_t)row0 * L.n;
  const uint32_t smb = smem_u32(sm);
  const int blocks = (rows + kBlockRows - 1) / kBlockRows;
  auto fetch = [&](int b) {
    stage.fetch(smb + (b & 1) * kBlockRows * SR * 4, p, L, act, b * kBlockRows, min(kBlockRows, rows - b * kBlockRows), h, hq, c0);
  };
  fetch(0);
  float* st = p.state + (((size_t)slot * p.H + h) * p.dv + c0 + warp * COLS) * dk + lane * 4;
  float4 S[ND / 4][NC];
  load_state<ND, NC>(S, st, p.pos[row0] == 0);
  const int col = warp * COLS + cl * NC;
  for (int b = 0; b < blocks; ++b) {
    if (b + 1 < blocks) {
      fetch(b + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int n = min(kBlockRows, rows - b * kBlockRows);
    for (int r = 0; r < n; ++r) {
      const float* row = sm + ((b & 1) * kBlockRows + r) * SR;
      const float4* q = reinterpret_cast<const float4*>(row) + dl;
      const float4* k = reinterpret_cast<const float4*>(row + dk) + dl;
      const float4* g = reinterpret_cast<const float4*>(row + 2 * dk) + dl;
      const float s1 = row[SR - 4], s2 = row[SR - 3];
      float v[NC], o[NC], a[NC];
#pragma unroll
      for (int j = 0; j < NC; ++j) {
        v[j] = row[3 * dk + col + j];
        o[j] = a[j] = 0.f;
      }
#pragma unroll
      for (int i = 0; i < ND / 4; ++i) {
        const float4 gv = g[i * LK], kv = k[i * LK], qv = q[i * LK];
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          if (DELTA) {
            S[i][j] = mul4(S[i][j], gv);
            a[j] = fdot4(S[i][j], kv, a[j]);
            o[j] = fdot4(S[i][j], qv, o[j]);
          } else {
            o[j] = fdot4(S[i][j], qv, o[j]);
            S[i][j] = axpy4(v[j], kv, mul4(S[i][j], gv));
          }
        }
      }
#pragma unroll
      for (int x = CL; x < 32; x <<= 1)
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          o[j] += __shfl_xor_sync(0xffffffffu, o[j], x);
          if (DELTA) a[j] += __shfl_xor_sync(0xffffffffu, a[j], x);
        }
      if (DELTA) {
#pragma unroll
        for (int j = 0; j < NC; ++j) {
          a[j] = s1 * (v[j] - a[j]);
          o[j] = fmaf(s2, a[j], o[j]);
        }
#pragma unroll
        for (int i = 0; i < ND / 4; ++i) {
          const float4 kv = k[i * LK];
#pragma unroll
          for (int j = 0; j < NC; ++j) S[i][j] = axpy4(a[j], kv, S[i][j]);
        }
      } else {
#pragma unroll
        for (int j = 0; j < NC; ++j) o[j] = fmaf(s1, v[j], o[j]);
      }
      const size_t at = (size_t)(row0 + b * kBlockRows + r) * (p.H * p.dv) + h * p.dv + c0 + col;
      if constexpr (FUSED) {
        float ssq = 0.f;
#pragma unroll
        for (int j = 0; j < NC; ++j) ssq += o[j] * o[j];
#pragma unroll
        for (int x = 1; x < CL; x <<= 1) ssq += __shfl_xor_sync(0xffffffffu, ssq, x);
        if (lane == 0) s_red[r & 1][warp] = ssq;
        __syncthreads();
        float tot = 0.f;
        for (int w = 0; w < warps; ++w) tot += s_red[r & 1][w];
        const float f = 1.f / sqrtf(tot / (float)p.vdim + p.eps);
        if (dl == 0) {
#pragma unroll
          for (int j = 0; j < NC; ++j) put(reinterpret_cast<T*>(p.out) + at + j, o[j] * f * p.norm[h * p.dv + c0 + col + j] * row[3 * dk + vb + col + j]);
        }
      } else if (dl == 0) {
#pragma unroll
        for (int j = 0; j < NC; ++j) p.o[at + j] = o[j];
      }
    }
    __syncthreads();       // the block's rows are read: the next fetch may overwrite them
  }
  store_state<ND, NC>(S, st);
}

// Segments: groups of four rows.  With a_t the product of a group's decays up to row t and b_s that of the decays after row s,
// the group needs the state at its start only through products with scaled rows, and one pass updates it:
//
//   delta rule   u_t = beta_t (v_t - S^T (a_t k_t) - sum_{s < t} c_ts u_s),   c_ts = (decays s + 1 .. t) k_s . k_t
//                o_t = S^T (a_t q_t) + sum_{s <= t} d_ts u_s,                 d_ts = (decays s + 1 .. t) k_s . q_t
//                S  <- a_3 S + sum_s (b_s k_s) u_s^T
//   time mixing  o_t = S^T (a_{t-1} q_t) + sum_{s < t} d_ts v_s + bonus_t v_t,  d_ts = (decays s + 1 .. t - 1) k_s . q_t
//                S  <- a_3 S + sum_s (b_s k_s) v_s^T
//
// Every factor is a product of decays (no quotients).  The CTA scales its staged rows in place, a thread per key dim.
template <int ND, int NC, bool DELTA>
__global__ void __launch_bounds__(128) channel_groups_kernel(const ScanParams p) {
  constexpr int LK = 8, CL = 4, dk = ND * LK, COLS = CL * NC, vb = 4 * COLS, G = kBlockRows / kGroup;
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(16) float s_pair[G][4][16], s_dots[G][2][16];     // per warp: partial sums; c and d of a group: [t][s]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, dl = lane / CL, cl = lane % CL;
  const int h = blockIdx.y, c0 = blockIdx.x * vb, hq = h / (p.H / p.Hq);
  pdl_launch_dependents();
  pdl_wait();
  int row0, rows, slot;
  if (!find_rows(p, row0, rows, slot)) return;
  commit_inputs(p, slot);
  const ActLayout L = act_layout(p.Hq, p.H, dk, p.dv);
  const Stage<dk, false> stage(vb);
  const int SR = stage.SR, SB = kBlockRows * SR + G * dk;      // a stage: rows, then a_3 of its groups
  const float* act = p.act + (size_t)row0 * L.n;
  const uint32_t smb = smem_u32(sm);
  const int blocks = (rows + kBlockRows - 1) / kBlockRows;
  auto fetch = [&](int b) {
    stage.fetch(smb + (b & 1) * SB * 4, p, L, act, b * kBlockRows, min(kBlockRows, rows - b * kBlockRows), h, hq, c0);
  };
  fetch(0);
  float* st = p.state + (((size_t)slot * p.H + h) * p.dv + c0 + warp * COLS) * dk + lane * 4;
  float4 S[ND / 4][NC];
  load_state<ND, NC>(S, st, p.pos[row0] == 0);
  const int col = warp * COLS + cl * NC;
  for (int b = 0; b < blocks; ++b) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();       // the block's rows are there, the block before is read
    if (b + 1 < blocks) fetch(b + 1);
    const int n = min(kBlockRows, rows - b * kBlockRows);
    float* base = sm + (b & 1) * SB;
#pragma unroll 1
    for (int gr = 0; gr < G; ++gr) {       // scaled rows, and the products of the group's rows with each other
      if (gr * kGroup >= n) break;
      float w[16];
#pragma unroll
      for (int e = 0; e < 16; ++e) w[e] = 0.f;
      for (int d = threadIdx.x; d < dk; d += 128) {
        float q[4], k[4], g[4];
        float* x = base + gr * kGroup * SR + d;
#pragma unroll
        for (int t = 0; t < 4; ++t) {
          const bool ok = gr * kGroup + t < n;       // rows past the end keep the state
          q[t] = ok ? x[t * SR] : 0.f;
          k[t] = ok ? x[t * SR + dk] : 0.f;
          g[t] = ok ? x[t * SR + 2 * dk] : 1.f;
        }
        float a = 1.f;
#pragma unroll
        for (int t = 0; t < 4; ++t) {
          if (DELTA) a *= g[t];
          x[t * SR] = a * q[t];
          if (DELTA) x[t * SR + dk] = a * k[t];
          if (!DELTA) a *= g[t];
        }
        base[kBlockRows * SR + gr * dk + d] = a;
        float c = 1.f;
#pragma unroll
        for (int t = 3; t >= 0; --t) {
          x[t * SR + 2 * dk] = c * k[t];
          c *= g[t];
        }
        // w: d_ts, s <= t, at 0 .. 9 in rows (time mixing: s < t); c_ts, s < t, at 10 .. 15
#pragma unroll
        for (int s = 0; s < 4; ++s) {
          float r = k[s];
          if (DELTA) w[s * (s + 1) / 2 + s] = fmaf(r, q[s], w[s * (s + 1) / 2 + s]);
#pragma unroll
          for (int t = s + 1; t < 4; ++t) {
            if (DELTA) r *= g[t];
            w[t * (t + 1) / 2 + s] = fmaf(r, q[t], w[t * (t + 1) / 2 + s]);
            if (DELTA) w[10 + t * (t - 1) / 2 + s] = fmaf(r, k[t], w[10 + t * (t - 1) / 2 + s]);
            else r *= g[t];
          }
        }
      }
      // sums over the warp, halving the values held per lane: lane l ends with value l >> 1
#pragma unroll
      for (int x = 16, m = 8; m >= 1; x >>= 1, m >>= 1)
#pragma unroll
        for (int e = 0; e < 8; ++e)
          if (e < m) {
            const bool up = lane & x;
            const float give = up ? w[e] : w[e + m], keep = up ? w[e + m] : w[e];
            w[e] = keep + __shfl_xor_sync(0xffffffffu, give, x);
          }
      w[0] += __shfl_xor_sync(0xffffffffu, w[0], 1);
      if (!(lane & 1)) s_pair[gr][warp][lane >> 1] = w[0];
    }
    __syncthreads();
    {                     // full 4 x 4 tables: d, then c
      const int gr = threadIdx.x >> 5, e = threadIdx.x & 31, t = (e >> 2) & 3, s = e & 3;
      const bool is_c = e >= 16;
      const int i = is_c ? 10 + t * (t - 1) / 2 + s : t * (t + 1) / 2 + s;
      const bool ok = DELTA ? (is_c ? s < t : s <= t) : !is_c && s < t;
      s_dots[gr][is_c][t * 4 + s] = ok ? s_pair[gr][0][i] + s_pair[gr][1][i] + s_pair[gr][2][i] + s_pair[gr][3][i] : 0.f;
    }
    __syncthreads();
    for (int gr = 0; gr * kGroup < n; ++gr) {
      const float* row = base + gr * kGroup * SR;
      float pq[4][NC], u[4][NC];
#pragma unroll
      for (int t = 0; t < 4; ++t)
#pragma unroll
        for (int j = 0; j < NC; ++j) pq[t][j] = u[t][j] = 0.f;
#pragma unroll
      for (int i = 0; i < ND / 4; ++i)
#pragma unroll
        for (int t = 0; t < 4; ++t) {
          const float4 qv = reinterpret_cast<const float4*>(row + t * SR)[i * LK + dl];
#pragma unroll
          for (int j = 0; j < NC; ++j) pq[t][j] = fdot4(S[i][j], qv, pq[t][j]);
          if (DELTA) {
            const float4 kv = reinterpret_cast<const float4*>(row + t * SR + dk)[i * LK + dl];
#pragma unroll
            for (int j = 0; j < NC; ++j) u[t][j] = fdot4(S[i][j], kv, u[t][j]);
          }
        }
      float v[4][NC];
#pragma unroll
      for (int t = 0; t < 4; ++t)
#pragma unroll
        for (int j = 0; j < NC; ++j) v[t][j] = gr * kGroup + t < n ? row[t * SR + 3 * dk + col + j] : 0.f;
      if (DELTA) {
#pragma unroll
        for (int x = CL; x < 32; x <<= 1)
#pragma unroll
          for (int t = 0; t < 4; ++t)
#pragma unroll
            for (int j = 0; j < NC; ++j) u[t][j] += __shfl_xor_sync(0xffffffffu, u[t][j], x);
#pragma unroll
        for (int t = 0; t < 4; ++t) {
          const float4 c = *reinterpret_cast<const float4*>(&s_dots[gr][1][t * 4]);
          const float beta = gr * kGroup + t < n ? row[t * SR + SR - 4] : 0.f;
#pragma unroll
          for (int j = 0; j < NC; ++j) {
            float r = v[t][j] - u[t][j];
            if (t > 0) r = fmaf(-c.x, u[0][j], r);
            if (t > 1) r = fmaf(-c.y, u[1][j], r);
            if (t > 2) r = fmaf(-c.z, u[2][j], r);
            u[t][j] = beta * r;
          }
        }
      } else {
#pragma unroll
        for (int t = 0; t < 4; ++t)
#pragma unroll
          for (int j = 0; j < NC; ++j) u[t][j] = v[t][j];
      }
      // the state after the group
      const float4* av = reinterpret_cast<const float4*>(base + kBlockRows * SR + gr * dk);
#pragma unroll
      for (int i = 0; i < ND / 4; ++i) {
        const float4 a = av[i * LK + dl];
#pragma unroll
        for (int j = 0; j < NC; ++j) S[i][j] = mul4(S[i][j], a);
#pragma unroll
        for (int t = 0; t < 4; ++t) {
          const float4 kv = reinterpret_cast<const float4*>(row + t * SR + 2 * dk)[i * LK + dl];
#pragma unroll
          for (int j = 0; j < NC; ++j) S[i][j] = axpy4(u[t][j], kv, S[i][j]);
        }
      }
      // read-outs: summed over the dim lanes so that lane dl ends with row dl & 3 (and column dl >> 2)
      const int t = dl & 3;
      float o[NC];
#pragma unroll
      for (int j = 0; j < NC; ++j) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float give = dl & 2 ? pq[e][j] : pq[e + 2][j], keep = dl & 2 ? pq[e + 2][j] : pq[e][j];
          pq[e][j] = keep + __shfl_xor_sync(0xffffffffu, give, 2 * CL);
        }
        const float give = dl & 1 ? pq[0][j] : pq[1][j], keep = dl & 1 ? pq[1][j] : pq[0][j];
        o[j] = keep + __shfl_xor_sync(0xffffffffu, give, CL);
      }
      int j = 0;
      float mine;
      if constexpr (NC == 2) {
        j = dl >> 2;
        mine = (j ? o[1] : o[0]) + __shfl_xor_sync(0xffffffffu, j ? o[0] : o[1], 4 * CL);
      } else {
        mine = o[0] + __shfl_xor_sync(0xffffffffu, o[0], 4 * CL);
      }
      const float4 d = *reinterpret_cast<const float4*>(&s_dots[gr][0][t * 4]);
      mine = fmaf(d.x, NC == 2 && j ? u[0][NC - 1] : u[0][0], mine);
      mine = fmaf(d.y, NC == 2 && j ? u[1][NC - 1] : u[1][0], mine);
      mine = fmaf(d.z, NC == 2 && j ? u[2][NC - 1] : u[2][0], mine);
      mine = fmaf(d.w, NC == 2 && j ? u[3][NC - 1] : u[3][0], mine);
      const int r = gr * kGroup + t;
      if (r < n && (NC == 2 || dl < 4)) {
        if (!DELTA) mine = fmaf(row[t * SR + SR - 4], row[t * SR + 3 * dk + col + j], mine);
        p.o[(size_t)(row0 + b * kBlockRows + r) * (p.H * p.dv) + h * p.dv + c0 + col + j] = mine;
      }
    }
  }
  store_state<ND, NC>(S, st);
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

// key dims of the kernels: 64, 128, 192, 256 with two value columns per lane, 384 and 512 with one
bool dk_ok(int dk) { return dk == 64 || dk == 128 || dk == 192 || dk == 256 || dk == 384 || dk == 512; }

template <typename F>
int launch_scan_kernel(F kernel, const ScanParams& p, dim3 grid, int threads, int smem, cudaStream_t st) {
  if (smem > 227 * 1024 - 4096) return -6;
  if (smem > 44 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
  }
  return b2_launch(kernel, grid, dim3(threads), smem, st, true, p);
}

template <int ND, int NC, bool DELTA, bool FUSED, typename T>
int launch_rows(const ScanParams& p, int seqs, cudaStream_t st) {
  const int warps = FUSED ? p.dv / (4 * NC) : 4, vb = warps * 4 * NC;
  const int smem = 2 * kBlockRows * (3 * ND * 8 + (FUSED ? 2 : 1) * vb + 4) * 4;
  return launch_scan_kernel(channel_rows_kernel<ND, NC, DELTA, FUSED, T>, p, dim3(p.dv / vb, p.H, seqs), warps * 32, smem, st);
}

template <int ND, int NC, bool DELTA>
int launch_groups(const ScanParams& p, int seqs, cudaStream_t st) {
  constexpr int vb = 16 * NC, smem = 2 * (kBlockRows * (3 * ND * 8 + vb + 4) + kBlockRows / kGroup * ND * 8) * 4;
  return launch_scan_kernel(channel_groups_kernel<ND, NC, DELTA>, p, dim3(p.dv / vb, p.H, seqs), 128, smem, st);
}

template <bool DELTA, typename T>
int launch_fused_dk(const ScanParams& p, int seqs, cudaStream_t st) {
  switch (p.dk) {
    case 64: return launch_rows<8, 2, DELTA, true, T>(p, seqs, st);
    case 128: return launch_rows<16, 2, DELTA, true, T>(p, seqs, st);
    case 192: return launch_rows<24, 2, DELTA, true, T>(p, seqs, st);
    case 256: return launch_rows<32, 2, DELTA, true, T>(p, seqs, st);
  }
  return -1;
}

template <bool DELTA>
int launch_scan_dk(const ScanParams& p, int seqs, cudaStream_t st) {
  if (p.segs) {
    switch (p.dk) {
      case 64: return launch_groups<8, 2, DELTA>(p, seqs, st);
      case 128: return launch_groups<16, 2, DELTA>(p, seqs, st);
      case 192: return launch_groups<24, 2, DELTA>(p, seqs, st);
      case 256: return launch_groups<32, 2, DELTA>(p, seqs, st);
      case 384: return launch_groups<48, 1, DELTA>(p, seqs, st);
      case 512: return launch_groups<64, 1, DELTA>(p, seqs, st);
    }
    return -1;
  }
  switch (p.dk) {
    case 64: return launch_rows<8, 2, DELTA, false, float>(p, seqs, st);
    case 128: return launch_rows<16, 2, DELTA, false, float>(p, seqs, st);
    case 192: return launch_rows<24, 2, DELTA, false, float>(p, seqs, st);
    case 256: return launch_rows<32, 2, DELTA, false, float>(p, seqs, st);
    case 384: return launch_rows<48, 1, DELTA, false, float>(p, seqs, st);
    case 512: return launch_rows<64, 1, DELTA, false, float>(p, seqs, st);
  }
  return -1;
}

template <int TP, int R, int QN, typename T>
int launch_delta_rows(const DeltaPrepParams& p, int tasks, cudaStream_t st) {
  return b2_launch(delta_prep_kernel<TP, R, QN, T>, dim3((tasks + 3) / 4, (p.M + R - 1) / R), dim3(128), 0, st, true, p);
}

template <int TP, typename T>
int launch_delta_prep(const DeltaPrepParams& p, int tasks, cudaStream_t st) {
  const int d = p.dk > p.dv ? p.dk : p.dv;
  if (d <= 128) return p.M > 64 ? launch_delta_rows<TP, 4, 1, T>(p, tasks, st) : launch_delta_rows<TP, 1, 1, T>(p, tasks, st);
  if (d <= 256) return p.M > 64 ? launch_delta_rows<TP, 2, 2, T>(p, tasks, st) : launch_delta_rows<TP, 1, 2, T>(p, tasks, st);
  return launch_delta_rows<TP, 1, 4, T>(p, tasks, st);
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
  const int tasks = Hq + H + (H * (dk + dv) + (lr ? 127 : 31)) / (lr ? 128 : 32);
  return f32 ? delta_prep_taps<float>(p, taps, tasks, (cudaStream_t)stream) : delta_prep_taps<__nv_bfloat16>(p, taps, tasks, (cudaStream_t)stream);
}

// part: r | k | v | g (H d columns each) | w1; lr: fp32 [lr_slices][M][H d], or null with w2 as above, [H d] rows
extern "C" int b2_wkv_prep(const float* part, int slices, int M, int N, int H, int d, int rank, const float* u, const float* w0,
                           const float* lr, int lr_slices, const void* w2, int kp, int ldw, float* act, int f32, void* stream) {
  if (M < 1 || slices < 1 || slices > 8 || H < 1 || !dk_ok(d) || N % 4 || kp % 64 || rank > kp || ldw < kp || ldw % 8 ||
      (!lr && !w2))
    return -1;
  WkvPrepParams p{part, slices, M, N, H, d, rank, u, w0, {lr, lr_slices, H * d, w2, kp, ldw}, act};
  const int tasks = (H + (H * d + (lr ? 127 : 31)) / (lr ? 128 : 32) + 3) / 4;
  cudaStream_t st = (cudaStream_t)stream;
  if (M > 64)
    return f32 ? b2_launch(wkv_prep_kernel<2, float>, dim3(tasks, (M + 1) / 2), dim3(128), 0, st, true, p)
               : b2_launch(wkv_prep_kernel<2, __nv_bfloat16>, dim3(tasks, (M + 1) / 2), dim3(128), 0, st, true, p);
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
    if (delta) return f32 ? launch_fused_dk<true, float>(p, seqs, st) : launch_fused_dk<true, __nv_bfloat16>(p, seqs, st);
    return f32 ? launch_fused_dk<false, float>(p, seqs, st) : launch_fused_dk<false, __nv_bfloat16>(p, seqs, st);
  }
  if (!raw) return -3;
  const int rc = delta ? launch_scan_dk<true>(p, seqs, st) : launch_scan_dk<false>(p, seqs, st);
  if (rc) return rc;
  const ActLayout L = act_layout(Hq, H, dk, dv);
  const dim3 grid((unsigned)(((long long)M * H + 7) / 8));
  return f32 ? b2_launch(channel_out_kernel<float>, grid, dim3(256), 0, st, true, (const float*)raw, act, L.n, L.z, norm, M, H, dv, vdim, eps, (float*)out)
             : b2_launch(channel_out_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, true, (const float*)raw, act, L.n, L.z, norm, M, H, dv, vdim, eps, (__nv_bfloat16*)out);
}

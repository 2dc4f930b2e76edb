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
//   channel_groups_kernel  the recurrence over prompt segments in fp32 arithmetic, four rows at a time
//   channel_pairs_kernel, channel_chunks_kernel  the same on the tensor cores, sixteen rows at a time: what does not involve the
//                        state for all chunks and heads at once, then the walk over the chunks
//   channel_out_kernel   head norm and output gate of what the scan left
//
// The prep kernels leave fp32 rows
//   q [Hq dk] | k [Hq dk] | decay [H dk] | v [H dv] | gate [H dv] | s1 [H] | s2 [H]     (both s padded to fours)
// with s1 = beta, s2 = k . q (delta rule) or s1 = bonus (time mixing).  Everything is fp32; models served in 32-bit use the
// same kernels.  A sequence's first row (position 0) starts from zeros whatever its slot holds.
//
// State of one slot: per head and tile of four value columns the elements in the order in which a warp holds them:
// [dk / 32][32 lanes][4 key dims].
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

// A warp holds the state of 4 NC value columns: lane = (dim lane dl = lane / 4, cl = lane % 4), column cl of each of its NC tiles, key
// dims (8 i + dl) 4 .. + 3.  The dim lanes are the upper lane bits: the four lanes that read the same 16 bytes of a shared row
// are then neighbours, which halves the wavefronts of the load.
template <int ND, int NC>
__device__ __forceinline__ void load_state(float4 (&S)[ND / 4][NC], const float* st, bool fresh) {
#pragma unroll
  for (int i = 0; i < ND / 4; ++i)
#pragma unroll
    for (int j = 0; j < NC; ++j)
      S[i][j] = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : __ldcg(reinterpret_cast<const float4*>(st + (j * (ND / 4) + i) * 128));
}
template <int ND, int NC>
__device__ __forceinline__ void store_state(const float4 (&S)[ND / 4][NC], float* st) {
#pragma unroll
  for (int i = 0; i < ND / 4; ++i)
#pragma unroll
    for (int j = 0; j < NC; ++j) *reinterpret_cast<float4*>(st + (j * (ND / 4) + i) * 128) = S[i][j];
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
  const int col = warp * COLS + cl;
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
        v[j] = row[3 * dk + col + 4 * j];
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
          for (int j = 0; j < NC; ++j) put(reinterpret_cast<T*>(p.out) + at + 4 * j, o[j] * f * p.norm[h * p.dv + c0 + col + 4 * j] * row[3 * dk + vb + col + 4 * j]);
        }
      } else if (dl == 0) {
#pragma unroll
        for (int j = 0; j < NC; ++j) p.o[at + 4 * j] = o[j];
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
// Eight warps: two halves of a CTA scale two groups at a time, then every warp walks all groups for its four value columns.
template <int ND, bool DELTA>
__global__ void __launch_bounds__(256) channel_groups_kernel(const ScanParams p) {
  constexpr int LK = 8, CL = 4, dk = ND * LK, vb = 8 * CL, G = kBlockRows / kGroup;
  extern __shared__ __align__(16) float sm[];
  __shared__ __align__(16) float s_pair[G][4][16], s_dots[G][2][16];     // per warp: partial sums; d and c of a group: [t][s]
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
  float* st = p.state + (((size_t)slot * p.H + h) * p.dv + c0 + warp * CL) * dk + lane * 4;
  float4 S[ND / 4][1];
  load_state<ND, 1>(S, st, p.pos[row0] == 0);
  const int col = warp * CL + cl;
  float* out = p.o + (size_t)row0 * (p.H * p.dv) + h * p.dv + c0 + col;
  for (int b = 0; b < blocks; ++b) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();       // the block's rows are there, the block before is read
    if (b + 1 < blocks) fetch(b + 1);
    const int n = min(kBlockRows, rows - b * kBlockRows);
    float* base = sm + (b & 1) * SB;
#pragma unroll 1
    for (int gr = warp >> 2; gr < G; gr += 2) {       // scaled rows, and the products of the group's rows with each other
      if (gr * kGroup >= n) break;
      float w[16];
#pragma unroll
      for (int e = 0; e < 16; ++e) w[e] = 0.f;
      for (int d = threadIdx.x & 127; d < dk; d += 128) {
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
      if (!(lane & 1)) s_pair[gr][warp & 3][lane >> 1] = w[0];
    }
    __syncthreads();
    if (threadIdx.x < 128) {      // full 4 x 4 tables: d, then c
      const int gr = threadIdx.x >> 5, e = threadIdx.x & 31, t = (e >> 2) & 3, s = e & 3;
      const bool is_c = e >= 16;
      const int i = is_c ? 10 + t * (t - 1) / 2 + s : t * (t + 1) / 2 + s;
      const bool ok = DELTA ? (is_c ? s < t : s <= t) : !is_c && s < t;
      s_dots[gr][is_c][t * 4 + s] = ok ? s_pair[gr][0][i] + s_pair[gr][1][i] + s_pair[gr][2][i] + s_pair[gr][3][i] : 0.f;
    }
    __syncthreads();
    for (int gr = 0; gr * kGroup < n; ++gr) {
      const float* row = base + gr * kGroup * SR;
      float pq[4], u[4], v[4], beta[4];
#pragma unroll
      for (int t = 0; t < 4; ++t) {
        const bool ok = gr * kGroup + t < n;
        pq[t] = u[t] = 0.f;
        v[t] = ok ? row[t * SR + 3 * dk + col] : 0.f;
        beta[t] = ok ? row[t * SR + SR - 4] : 0.f;          // time mixing: the bonus
      }
#pragma unroll
      for (int i = 0; i < ND / 4; ++i)
#pragma unroll
        for (int t = 0; t < 4; ++t) {
          if (DELTA) u[t] = fdot4(S[i][0], reinterpret_cast<const float4*>(row + t * SR + dk)[i * LK + dl], u[t]);
          pq[t] = fdot4(S[i][0], reinterpret_cast<const float4*>(row + t * SR)[i * LK + dl], pq[t]);
        }
      if (DELTA) {
#pragma unroll
        for (int x = CL; x < 32; x <<= 1)
#pragma unroll
          for (int t = 0; t < 4; ++t) u[t] += __shfl_xor_sync(0xffffffffu, u[t], x);
#pragma unroll
        for (int t = 0; t < 4; ++t) {
          const float4 c = *reinterpret_cast<const float4*>(&s_dots[gr][1][t * 4]);
          float r = v[t] - u[t];
          if (t > 0) r = fmaf(-c.x, u[0], r);
          if (t > 1) r = fmaf(-c.y, u[1], r);
          if (t > 2) r = fmaf(-c.z, u[2], r);
          u[t] = beta[t] * r;
        }
      } else {
#pragma unroll
        for (int t = 0; t < 4; ++t) u[t] = v[t];
      }
      // the state after the group
      const float4* av = reinterpret_cast<const float4*>(base + kBlockRows * SR + gr * dk);
#pragma unroll
      for (int i = 0; i < ND / 4; ++i) {
        float4 x = mul4(S[i][0], av[i * LK + dl]);
#pragma unroll
        for (int t = 0; t < 4; ++t) x = axpy4(u[t], reinterpret_cast<const float4*>(row + t * SR + 2 * dk)[i * LK + dl], x);
        S[i][0] = x;
      }
      // read-outs: summed over the dim lanes so that lane dl ends with row dl & 3
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float give = dl & 2 ? pq[e] : pq[e + 2], keep = dl & 2 ? pq[e + 2] : pq[e];
        pq[e] = keep + __shfl_xor_sync(0xffffffffu, give, 2 * CL);
      }
      const float give = dl & 1 ? pq[0] : pq[1], keep = dl & 1 ? pq[1] : pq[0];
      float o = keep + __shfl_xor_sync(0xffffffffu, give, CL);
      o += __shfl_xor_sync(0xffffffffu, o, 4 * CL);
      const int t = dl & 3, r = gr * kGroup + t;
      const float4 d = *reinterpret_cast<const float4*>(&s_dots[gr][0][t * 4]);
      o = fmaf(d.x, u[0], o);
      o = fmaf(d.y, u[1], o);
      o = fmaf(d.z, u[2], o);
      o = fmaf(d.w, u[3], o);
      if (!DELTA) o = fmaf(t == 0 ? beta[0] : t == 1 ? beta[1] : t == 2 ? beta[2] : beta[3], t == 0 ? v[0] : t == 1 ? v[1] : t == 2 ? v[2] : v[3], o);
      if (r < n && dl < 4) out[(size_t)(b * kBlockRows + r) * (p.H * p.dv)] = o;
    }
  }
  store_state<ND, 1>(S, st);
}

// ------------------------------------------------------------------ segments on the tensor cores
// Chunks of sixteen rows, in the notation of the groups above.  With the rows' writes U and the state S0 at the chunk's start
//   delta rule   (I + diag(beta) C) U = diag(beta) (V - Kp S0),  so  U = Wv - W S0   with  W = (I + diag(beta) C)^-1 diag(beta) Kp
//                and Wv likewise from V;   Kp, Qp: rows a_t k_t, a_t q_t
//   time mixing  U = V;  Qp: rows a_{t-1} q_t;  the bonus is the diagonal of D
//   both         O = Qp S0 + D U,   S <- diag(a_15) S0 + Ks^T U,   Ks: rows b_s k_s
// W, Qp, Ks and D enter their products as two bf16 limbs, as do the state and U; a product of two such keeps all but the
// smallest of its four terms.
constexpr int CR = 16;                                    // rows of a chunk
constexpr int kLdd = 24, kLdv = 20;                       // row strides of D (bf16) and of Wv^T (fp32)

// operand block of a (chunk, head): [W hi | W lo |] Q hi | Q lo | Ks hi | Ks lo ([16][dk + 8] bf16 each), a_15 [dk] fp32, D hi | lo
// [16][24] bf16, then Wv^T [dv][20] fp32
template <int KB, bool DELTA>
struct Block {
  static constexpr int dk = KB * 64, LDK = dk + 8, IMG = CR * LDK * 2;
  static constexpr int W = 0, Q = DELTA ? 2 * IMG : 0, K = Q + 2 * IMG, A = K + 2 * IMG, D = A + dk * 4, V = D + 2 * CR * kLdd * 2;
  static constexpr int SLICE = 64 * kLdv * 4;             // Wv^T of 64 value columns
  static constexpr int STAGE = V + SLICE, NST = KB <= 2 ? 4 : 3;
  static constexpr int SMEM = NST * STAGE + 64 + 128;
  static_assert(IMG % 16 == 0 && V % 16 == 0 && STAGE % 16 == 0, "bulk copies move multiples of 16 bytes");
  static_assert(SMEM <= 227 * 1024, "shared memory of one CTA");
  __host__ __device__ static constexpr size_t bytes(int dv) { return V + (size_t)dv * kLdv * 4; }
};

struct ChunkParams {
  ScanParams s;
  uint8_t* ws;             // [16-row chunks][H] blocks; a segment's first chunk is four times its `first chunk` word
};

__device__ __forceinline__ void limbs(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - bf16_lo(hi), y - bf16_hi(hi));
}

template <int KB, bool DELTA>
__global__ void __launch_bounds__(128) channel_pairs_kernel(const ChunkParams cp) {
  using B = Block<KB, DELTA>;
  constexpr int dk = KB * 64, NQ = (dk + 127) / 128;
  extern __shared__ __align__(16) float sm[];             // q | k | decay, [16][dk] each
  __shared__ __align__(16) float s_c[CR][CR], s_d[CR][CR], s_s1[CR];
  const ScanParams& p = cp.s;
  const int h = blockIdx.y, hq = h / (p.H / p.Hq), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int* seg = p.segs + blockIdx.z * 4;
  const int n = min(CR, seg[1] - (int)blockIdx.x * CR);
  if (n <= 0) return;
  const ActLayout L = act_layout(p.Hq, p.H, dk, p.dv);
  const float* act = p.act + (size_t)(seg[0] + blockIdx.x * CR) * L.n;
  uint8_t* blk = cp.ws + ((size_t)(4 * seg[3] + blockIdx.x) * p.H + h) * B::bytes(p.dv);
  float *sq = sm, *sk = sm + CR * dk, *sg = sm + 2 * CR * dk;
#pragma unroll
  for (int i = 0; i < 3 * CR * dk / 4 / 128; ++i) {
    const int e = (i * 128 + tid) * 4, which = e / (CR * dk), r = (e / dk) % CR, d = e % dk;
    const int col = which == 0 ? L.q + hq * dk : which == 1 ? L.k + hq * dk : L.g + h * dk;
    const float pad = which == 2 ? 1.f : 0.f;             // rows past the end keep the state
    *reinterpret_cast<float4*>(sm + e) = r < n ? __ldcg(reinterpret_cast<const float4*>(act + (size_t)r * L.n + col + d))
                                               : make_float4(pad, pad, pad, pad);
  }
  if (tid < CR) s_s1[tid] = tid < n ? act[(size_t)tid * L.n + L.s1 + h] : 0.f;
  __syncthreads();
  // products of the rows with each other: a warp takes four rows s, lanes the key dims; sums over the warp leave value l in
  // lane l (c_ts: t, d_ts: 16 + t)
  for (int i = 0; i < 4; ++i) {
    const int s = i == 0 ? warp : i == 1 ? 7 - warp : i == 2 ? 8 + warp : 15 - warp;
    float v[32];
#pragma unroll
    for (int e = 0; e < 32; ++e) v[e] = 0.f;
#pragma unroll
    for (int u = 0; u < NQ; ++u) {
      const int d = (u * 32 + lane) * 4;
      if (d >= dk) continue;
      float4 r = *reinterpret_cast<const float4*>(sk + s * dk + d);
#pragma unroll
      for (int t = 0; t < CR; ++t) {
        if (t < s) continue;
        const float4 g = *reinterpret_cast<const float4*>(sg + t * dk + d);
        const float4 q = *reinterpret_cast<const float4*>(sq + t * dk + d);
        if (DELTA) {
          if (t > s) {
            r = mul4(r, g);
            v[t] = fdot4(r, *reinterpret_cast<const float4*>(sk + t * dk + d), v[t]);
          }
          v[16 + t] = fdot4(r, q, v[16 + t]);
        } else if (t > s) {
          v[16 + t] = fdot4(r, q, v[16 + t]);
          r = mul4(r, g);
        }
      }
    }
#pragma unroll
    for (int x = 16; x >= 1; x >>= 1)
#pragma unroll
      for (int e = 0; e < 16; ++e)
        if (e < x) {
          const bool up = lane & x;
          const float give = up ? v[e] : v[e + x], keep = up ? v[e + x] : v[e];
          v[e] = keep + __shfl_xor_sync(0xffffffffu, give, x);
        }
    if (lane < 16) s_c[lane][s] = v[0];
    else s_d[lane - 16][s] = !DELTA && lane - 16 == s ? s_s1[s] : v[0];
  }
  __syncthreads();
  if (tid < CR * CR / 2) {             // D's limbs
    const int t = tid >> 3, s = (tid & 7) * 2;
    uint32_t hi, lo;
    limbs(s_d[t][s], s_d[t][s + 1], hi, lo);
    uint32_t* d = reinterpret_cast<uint32_t*>(blk + B::D) + (t * kLdd + s) / 2;
    d[0] = hi;
    d[CR * kLdd / 2] = lo;
  }
  // two columns per thread: of the keys (scaled rows, W), then of the values
  for (int c = tid; c < (dk + p.dv) / 2; c += 128) {
    const bool key = c < dk / 2;
    const int d = 2 * (key ? c : c - dk / 2);
    float2 x[CR];
    if (key) {
      float2 a = make_float2(1.f, 1.f);
#pragma unroll
      for (int t = 0; t < CR; ++t) {
        const float2 g = *reinterpret_cast<const float2*>(sg + t * dk + d);
        const float2 q = *reinterpret_cast<const float2*>(sq + t * dk + d), k = *reinterpret_cast<const float2*>(sk + t * dk + d);
        if (DELTA) a = make_float2(a.x * g.x, a.y * g.y);
        uint32_t hi, lo;
        limbs(a.x * q.x, a.y * q.y, hi, lo);
        uint32_t* o = reinterpret_cast<uint32_t*>(blk + B::Q) + (t * B::LDK + d) / 2;
        o[0] = hi;
        o[B::IMG / 4] = lo;
        x[t] = make_float2(a.x * k.x, a.y * k.y);
        if (!DELTA) a = make_float2(a.x * g.x, a.y * g.y);
      }
      *reinterpret_cast<float2*>(blk + B::A + d * 4) = a;
      float2 b = make_float2(1.f, 1.f);
#pragma unroll
      for (int t = CR - 1; t >= 0; --t) {
        const float2 g = *reinterpret_cast<const float2*>(sg + t * dk + d), k = *reinterpret_cast<const float2*>(sk + t * dk + d);
        uint32_t hi, lo;
        limbs(b.x * k.x, b.y * k.y, hi, lo);
        uint32_t* o = reinterpret_cast<uint32_t*>(blk + B::K) + (t * B::LDK + d) / 2;
        o[0] = hi;
        o[B::IMG / 4] = lo;
        b = make_float2(b.x * g.x, b.y * g.y);
      }
      if (!DELTA) continue;
    } else {
#pragma unroll
      for (int t = 0; t < CR; ++t)
        x[t] = t < n ? __ldcg(reinterpret_cast<const float2*>(act + (size_t)t * L.n + L.v + h * p.dv + d)) : make_float2(0.f, 0.f);
    }
    if (DELTA) {                       // forward substitution
#pragma unroll
      for (int t = 0; t < CR; ++t) {
        float2 y = x[t];
#pragma unroll
        for (int s = 0; s < t; ++s) y = make_float2(fmaf(-s_c[t][s], x[s].x, y.x), fmaf(-s_c[t][s], x[s].y, y.y));
        x[t] = make_float2(s_s1[t] * y.x, s_s1[t] * y.y);
      }
    }
    if (key) {
#pragma unroll
      for (int t = 0; t < CR; ++t) {
        uint32_t hi, lo;
        limbs(x[t].x, x[t].y, hi, lo);
        uint32_t* o = reinterpret_cast<uint32_t*>(blk + B::W) + (t * B::LDK + d) / 2;
        o[0] = hi;
        o[B::IMG / 4] = lo;
      }
    } else {
      float4* o = reinterpret_cast<float4*>(blk + B::V) + d * (kLdv / 4);
#pragma unroll
      for (int t = 0; t < CR; t += 4) {
        o[t / 4] = make_float4(x[t].x, x[t + 1].x, x[t + 2].x, x[t + 3].x);
        o[kLdv / 4 + t / 4] = make_float4(x[t].y, x[t + 1].y, x[t + 2].y, x[t + 3].y);
      }
    }
  }
}

__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_a(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  mma_bf16_16816(c, a[0], a[1], a[2], a[3], b0, b1);
}

// grid (value blocks of 64, heads, segments), four warps.  A warp keeps S^T of its 16 value columns in MMA accumulators for the whole
// walk; products have the value dimension as M, so accumulators become A operands in registers and the warps exchange nothing.
template <int KB, bool DELTA>
__global__ void __launch_bounds__(128) channel_chunks_kernel(const ChunkParams cp) {
  using B = Block<KB, DELTA>;
  constexpr int dk = KB * 64, NST = B::NST;
  extern __shared__ __align__(128) uint8_t smem_b[];
  const ScanParams& p = cp.s;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int h = blockIdx.y, c0 = blockIdx.x * 64;
  const uint32_t base = smem_u32(smem_b), bars = base + NST * B::STAGE;
  if (tid == 0) {
    for (int i = 0; i < NST; ++i) mbar_init(bars + 8 * i, 1);
    mbar_fence_init();
  }
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait();
  const int* seg = p.segs + blockIdx.z * 4;
  const int row0 = seg[0], rows = seg[1], slot = seg[2], chunks = (rows + CR - 1) / CR;
  commit_inputs(p, slot);
  const uint8_t* ws = cp.ws + ((size_t)4 * seg[3] * p.H + h) * B::bytes(p.dv);
  const size_t step = (size_t)p.H * B::bytes(p.dv);
  auto fetch = [&](int c) {
    const uint32_t dst = base + (c % NST) * B::STAGE, bar = bars + 8 * (c % NST);
    const uint8_t* src = ws + (size_t)c * step;
    mbar_expect_tx(bar, B::STAGE);
    bulk_g2s(dst, src, B::V, bar);
    bulk_g2s(dst + B::V, src + B::V + (size_t)c0 * kLdv * 4, B::SLICE, bar);
  };
  int issued = min(NST, chunks);
  if (tid == 0)
    for (int c = 0; c < issued; ++c) fetch(c);
  // st[j]: key dims 8 j + 2 t, + 1 of value column vc ([0], [1]) and of column vc + 8 ([2], [3])
  float st[dk / 8][4];
  const int vc = 16 * warp + g;
  float* sp = p.state + (((size_t)slot * p.H + h) * p.dv + c0) * dk;
  auto place = [&](int d, int col) { return (col >> 2) * 4 * dk + (d >> 5) * 128 + (((d >> 2) & 7) * 4 + (col & 3)) * 4 + (d & 3); };
  const bool fresh = p.pos[row0] == 0;
#pragma unroll
  for (int j = 0; j < dk / 8; ++j)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const float2 v = fresh ? make_float2(0.f, 0.f) : __ldcg(reinterpret_cast<const float2*>(sp + place(8 * j + 2 * t, vc + 8 * hf)));
      st[j][2 * hf] = v.x;
      st[j][2 * hf + 1] = v.y;
    }
  // ldmatrix lanes: B rows [n][k] of two n tiles, and rows [k][n] read transposed
  const uint32_t nk = (uint32_t)((((lane & 7) + ((lane >> 4) << 3)) * B::LDK + (((lane >> 3) & 1) << 3)) * 2);
  const uint32_t nd = (uint32_t)((((lane & 7) + ((lane >> 4) << 3)) * kLdd + (((lane >> 3) & 1) << 3)) * 2);
  const uint32_t kn = (uint32_t)((((lane & 7) + (((lane >> 3) & 1) << 3)) * B::LDK + ((lane >> 4) << 3)) * 2);
  bool ok = true;
  for (int c = 0; c < chunks; ++c) {
    const uint32_t sb = base + (c % NST) * B::STAGE;
    const uint8_t* sbp = smem_b + (c % NST) * B::STAGE;
    ok = mbar_wait(bars + 8 * (c % NST), (c / NST) & 1, ERR_GDN_WAIT);
    if (!__syncthreads_and(ok)) {      // a copy gave up: wait (bounded) for those in flight, leave the state alone
      if (tid == 0)
        for (int i = c; i < issued; ++i) mbar_wait(bars + 8 * (i % NST), (i / NST) & 1, ERR_GDN_WAIT);
      return;
    }
    // the state against W and Q: [16 value columns][16 rows]; small terms in sums of their own
    float r1[2][4] = {}, r2[2][4] = {}, e1[2][4] = {}, e2[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < dk / 16; ++kk) {
      uint32_t ah[4], al[4], qh[4], ql[4];
      limbs(st[2 * kk][0], st[2 * kk][1], ah[0], al[0]);
      limbs(st[2 * kk][2], st[2 * kk][3], ah[1], al[1]);
      limbs(st[2 * kk + 1][0], st[2 * kk + 1][1], ah[2], al[2]);
      limbs(st[2 * kk + 1][2], st[2 * kk + 1][3], ah[3], al[3]);
      if (DELTA) {
        uint32_t wh[4], wl[4];
        ldsm_x4(sb + B::W + nk + 32 * kk, wh);
        ldsm_x4(sb + B::W + B::IMG + nk + 32 * kk, wl);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          mma_a(r1[u], ah, wh[2 * u], wh[2 * u + 1]);
          mma_a(e1[u], al, wh[2 * u], wh[2 * u + 1]);
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) mma_a(e1[u], ah, wl[2 * u], wl[2 * u + 1]);
      }
      ldsm_x4(sb + B::Q + nk + 32 * kk, qh);
      ldsm_x4(sb + B::Q + B::IMG + nk + 32 * kk, ql);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        mma_a(r2[u], ah, qh[2 * u], qh[2 * u + 1]);
        mma_a(e2[u], al, qh[2 * u], qh[2 * u + 1]);
      }
#pragma unroll
      for (int u = 0; u < 2; ++u) mma_a(e2[u], ah, ql[2 * u], ql[2 * u + 1]);
    }
    // U^T as an A operand over the chunk's rows
    uint32_t uh[4], ul[4];
    const float* wv = reinterpret_cast<const float*>(sbp + B::V);
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        float2 v = *reinterpret_cast<const float2*>(wv + (vc + 8 * hf) * kLdv + 8 * u + 2 * t);
        if (DELTA) {
          v.x -= r1[u][2 * hf] + e1[u][2 * hf];
          v.y -= r1[u][2 * hf + 1] + e1[u][2 * hf + 1];
        }
        limbs(v.x, v.y, uh[2 * u + hf], ul[2 * u + hf]);
      }
    {
      uint32_t dh[4], dl[4];
      ldsm_x4(sb + B::D + nd, dh);
      ldsm_x4(sb + B::D + CR * kLdd * 2 + nd, dl);
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        mma_a(r2[u], uh, dh[2 * u], dh[2 * u + 1]);
        mma_a(e2[u], ul, dh[2 * u], dh[2 * u + 1]);
      }
#pragma unroll
      for (int u = 0; u < 2; ++u) mma_a(e2[u], uh, dl[2 * u], dl[2 * u + 1]);
    }
    // the state after the chunk
    const float* av = reinterpret_cast<const float*>(sbp + B::A);
#pragma unroll
    for (int j = 0; j < dk / 8; ++j) {
      const float2 a = *reinterpret_cast<const float2*>(av + 8 * j + 2 * t);
      st[j][0] *= a.x; st[j][1] *= a.y; st[j][2] *= a.x; st[j][3] *= a.y;
    }
#pragma unroll
    for (int jj = 0; jj < dk / 16; ++jj) {
      uint32_t kh[4], kl[4];
      ldsm_x4_trans(sb + B::K + kn + 32 * jj, kh);
      ldsm_x4_trans(sb + B::K + B::IMG + kn + 32 * jj, kl);
#pragma unroll
      for (int u = 0; u < 2; ++u) mma_a(st[2 * jj + u], ul, kh[2 * u], kh[2 * u + 1]);
#pragma unroll
      for (int u = 0; u < 2; ++u) mma_a(st[2 * jj + u], uh, kl[2 * u], kl[2 * u + 1]);
#pragma unroll
      for (int u = 0; u < 2; ++u) mma_a(st[2 * jj + u], uh, kh[2 * u], kh[2 * u + 1]);
    }
    float* o = p.o + (size_t)(row0 + c * CR) * (p.H * p.dv) + h * p.dv + c0 + vc;
    const int n = rows - c * CR;
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = 8 * u + 2 * t + (e & 1);
        if (r < n) o[(size_t)r * (p.H * p.dv) + 8 * (e >> 1)] = r2[u][e] + e2[u][e];
      }
    __syncthreads();       // every warp is done with the stage
    if (c + NST < chunks) {
      if (tid == 0) fetch(c + NST);
      issued = c + NST + 1;
    }
  }
#pragma unroll
  for (int j = 0; j < dk / 8; ++j)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf)
      *reinterpret_cast<float2*>(sp + place(8 * j + 2 * t, vc + 8 * hf)) = make_float2(st[j][2 * hf], st[j][2 * hf + 1]);
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
int launch_scan_kernel(F kernel, const ScanParams& p, dim3 grid, int threads, int smem, cudaStream_t st, bool pdl = true) {
  if (smem > 227 * 1024 - 4096) return -6;
  if (smem > 44 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
  }
  return b2_launch(kernel, grid, dim3(threads), smem, st, pdl, p);
}

template <int ND, int NC, bool DELTA, bool FUSED, typename T>
int launch_rows(const ScanParams& p, int seqs, cudaStream_t st) {
  const int warps = FUSED ? p.dv / (4 * NC) : 4, vb = warps * 4 * NC;
  const int smem = 2 * kBlockRows * (3 * ND * 8 + (FUSED ? 2 : 1) * vb + 4) * 4;
  return launch_scan_kernel(channel_rows_kernel<ND, NC, DELTA, FUSED, T>, p, dim3(p.dv / vb, p.H, seqs), warps * 32, smem, st);
}

// not started while the kernel before still runs: its few, long CTAs would gather on the SMs that happen to be free
template <int ND, bool DELTA>
int launch_groups(const ScanParams& p, int seqs, cudaStream_t st) {
  constexpr int vb = 32, smem = 2 * (kBlockRows * (3 * ND * 8 + vb + 4) + kBlockRows / kGroup * ND * 8) * 4;
  return launch_scan_kernel(channel_groups_kernel<ND, DELTA>, p, dim3(p.dv / vb, p.H, seqs), 256, smem, st, false);
}

template <int KB, bool DELTA>
int launch_chunks(const ChunkParams& p, int n_segs, int most, size_t ws_bytes, int chunks, cudaStream_t st) {
  using B = Block<KB, DELTA>;
  if (ws_bytes < (size_t)chunks * p.s.H * B::bytes(p.s.dv)) return -7;
  constexpr int psm = 3 * CR * KB * 64 * 4;
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(channel_chunks_kernel<KB, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, B::SMEM);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(channel_pairs_kernel<KB, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, psm);
    if (e != cudaSuccess) return (int)e;
    configured[dev & 63] = true;
  }
  int rc = b2_launch(channel_pairs_kernel<KB, DELTA>, dim3(most, p.s.H, n_segs), dim3(128), psm, st, true, p);
  if (rc) return rc;
  return b2_launch(channel_chunks_kernel<KB, DELTA>, dim3(p.s.dv / 64, p.s.H, n_segs), dim3(128), B::SMEM, st, false, p);     // as launch_groups
}

template <bool DELTA>
int launch_chunks_dk(const ChunkParams& p, int n_segs, int most, size_t ws_bytes, int chunks, cudaStream_t st) {
  switch (p.s.dk) {
    case 64: return launch_chunks<1, DELTA>(p, n_segs, most, ws_bytes, chunks, st);
    case 128: return launch_chunks<2, DELTA>(p, n_segs, most, ws_bytes, chunks, st);
    case 192: return launch_chunks<3, DELTA>(p, n_segs, most, ws_bytes, chunks, st);
    case 256: return launch_chunks<4, DELTA>(p, n_segs, most, ws_bytes, chunks, st);
  }
  return -1;
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
      case 64: return launch_groups<8, DELTA>(p, seqs, st);
      case 128: return launch_groups<16, DELTA>(p, seqs, st);
      case 192: return launch_groups<24, DELTA>(p, seqs, st);
      case 256: return launch_groups<32, DELTA>(p, seqs, st);
      case 384: return launch_groups<48, DELTA>(p, seqs, st);
      case 512: return launch_groups<64, DELTA>(p, seqs, st);
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

// bytes of a (16-row chunk, head) operand block of the tensor-core form; 0: the sizes are outside it
extern "C" int b2_channel_block_bytes(int delta, int dk, int dv) {
  switch (dk * 2 + (delta ? 1 : 0)) {
    case 128: return (int)Block<1, false>::bytes(dv);
    case 129: return (int)Block<1, true>::bytes(dv);
    case 256: return (int)Block<2, false>::bytes(dv);
    case 257: return (int)Block<2, true>::bytes(dv);
    case 384: return (int)Block<3, false>::bytes(dv);
    case 385: return (int)Block<3, true>::bytes(dv);
    case 512: return (int)Block<4, false>::bytes(dv);
    case 513: return (int)Block<4, true>::bytes(dv);
  }
  return 0;
}

// The recurrence over prepared rows.  segs null: rows 0 .. M - 1, a sequence per run of equal `req`; else n_segs x 4 ints
// (first row, rows, slot, first 64-row chunk; `chunks` such chunks in all, `most` in one segment).  With `ws` (segments; chunks x 4 x
// H blocks of b2_channel_block_bytes) on the tensor cores.  out [rows][H dv]; raw: fp32 of the same shape, unused where b2_channel_fused says so and
// segs is null.  delta 1: delta rule, 0: time mixing.
extern "C" int b2_channel_scan(const float* act, int delta, int M, int Hq, int H, int dk, int dv, int vdim, const int* req, const int* pos,
                               const int* segs, int n_segs, int chunks, int most, float* state, const float* conv_next, float* conv_state,
                               int conv_elems, const float* norm, float eps, void* ws, long long ws_bytes, float* raw, void* out, int f32,
                               void* stream) {
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
  int rc;
  if (segs && ws) {
    if ((uintptr_t)ws & 15) return -8;
    const ChunkParams cp{p, (uint8_t*)ws};
    rc = delta ? launch_chunks_dk<true>(cp, n_segs, 4 * most, (size_t)ws_bytes, 4 * chunks, st)
               : launch_chunks_dk<false>(cp, n_segs, 4 * most, (size_t)ws_bytes, 4 * chunks, st);
  } else {
    rc = delta ? launch_scan_dk<true>(p, seqs, st) : launch_scan_dk<false>(p, seqs, st);
  }
  if (rc) return rc;
  const ActLayout L = act_layout(Hq, H, dk, dv);
  const dim3 grid((unsigned)(((long long)M * H + 7) / 8));
  return f32 ? b2_launch(channel_out_kernel<float>, grid, dim3(256), 0, st, true, (const float*)raw, act, L.n, L.z, norm, M, H, dv, vdim, eps, (float*)out)
             : b2_launch(channel_out_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, true, (const float*)raw, act, L.n, L.z, norm, M, H, dv, vdim, eps, (__nv_bfloat16*)out);
}

B2_DEFINE_STATUS(channel)

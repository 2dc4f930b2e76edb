// Residual with a norm on both sides of every sublayer, in one pass over the rows:
//
//   y  = sum_s f_s N_s(source s)       what a sublayer left: one source, or two mixers' results, each through its own RMS norm
//   x' = x + G(y) o post               G: every one of `groups` equal parts of a row by its own root mean square
//   h  = G(x') o next                  what the next sublayer reads, rounded
//
// A source is a linear's split-K slices, or a mixture-of-experts row's weighted slots (slices per slot, or rows of the
// expert-sorted buffer), folded here in a fixed order; everything is fp32.  The first call of a step has the embedding rows as
// its source (`vocab` > 0: value rows are tokens), no residual and no post norm; the last one leaves the head's input and no
// residual.
//
// Two forms.  Groups of whole 128s: a CTA keeps a row in registers, every warp a run of 128 columns at a time, and meets once per
// norm; few rows get a thread per four columns.  Any other size goes through shared memory; few rows are then shared by a cluster
// of up to 8 CTAs, which exchange their sums of squares through distributed shared memory.
#include "common.cuh"

#include <cooperative_groups.h>

using namespace b2;
namespace cg = cooperative_groups;

namespace {

constexpr int kThreads = 256, kWarps = kThreads / 32;
constexpr int kTerms = 256;     // slots x slices of a source's row
constexpr int kGroups = 512;

}  // namespace

// host structure (ops/sandwich.py)
struct B2Source {
  const void* y;             // fp32 (or bf16) values
  const int* row_of;         // value row of (m, slot); null: m * slots + slot
  const float* slot_w;       // [M][slots]; null: every slot counts once
  long long slice, row;      // elements between split-K slices of a value row, between value rows
  int slots, slices, bf16;
  float factor;
  const float* norm;         // [ld] weight of an RMS norm over the row, or null
};

namespace {

struct SandwichParams {
  B2Source src[2];
  int n_src;
  int vocab;                 // > 0: the first source's value rows are tokens; others than 0 .. vocab - 1 set the flag and read row 0
  int* flag;
  int M, width, ld, groups, size;      // size: columns of a group
  float eps;
  const float *post, *next;  // [ld], padding zero; post null: no norm of y
  const float* x_in;         // [M][ld], or null
  float* x_out;              // [M][ld], or null
  void* h;                   // [M][ld]
  int h_f32;
};

__device__ __forceinline__ float4 value4(const B2Source& s, long long at) {
  if (!s.bf16) return __ldcg(reinterpret_cast<const float4*>(reinterpret_cast<const float*>(s.y) + at));
  const uint2 r = __ldcg(reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(s.y) + at));
  return make_float4(bf16_lo(r.x), bf16_hi(r.x), bf16_lo(r.y), bf16_hi(r.y));
}

// Sums of squares of the row's groups: those of this CTA's columns [c0, c1) of `vals` (indexed by column) to `stat`, then all of
// the cluster's together, as 1 / root mean square, to `inv`.
template <int CS>
__device__ __forceinline__ void group_stats(const float* vals, int c0, int c1, int groups, int size, float eps, float* red, float* stat,
                                            float* inv) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (groups < kWarps) {         // several warps per group
    const int per = kWarps / groups, g = warp / per, w = warp % per;
    float s = 0.f;
    if (g < groups) {
      const int lo = max(c0, g * size), hi = min(c1, (g + 1) * size);
      for (int c = lo + w * 32 + lane; c < hi; c += per * 32) s = fmaf(vals[c], vals[c], s);
    }
    s = warp_sum(s);
    if (lane == 0) red[warp] = s;
    __syncthreads();
    if (threadIdx.x < groups) {
      float a = 0.f;
      for (int i = 0; i < per; ++i) a += red[threadIdx.x * per + i];
      stat[threadIdx.x] = a;
    }
  } else {
    for (int g = warp; g < groups; g += kWarps) {
      const int lo = max(c0, g * size), hi = min(c1, (g + 1) * size);
      float s = 0.f;
      for (int c = lo + lane; c < hi; c += 32) s = fmaf(vals[c], vals[c], s);
      s = warp_sum(s);
      if (lane == 0) stat[g] = s;
    }
  }
  if (CS > 1) cg::this_cluster().sync();
  else __syncthreads();
  for (int g = threadIdx.x; g < groups; g += kThreads) {
    float a = 0.f;
    if (CS > 1) {
      cg::cluster_group cl = cg::this_cluster();
#pragma unroll
      for (int i = 0; i < CS; ++i) a += *cl.map_shared_rank(stat + g, i);
    } else {
      a = stat[g];
    }
    inv[g] = 1.f / sqrtf(a / (float)size + eps);
  }
  __syncthreads();
}

// factor of column c's group; padding columns are zero whatever it is
__device__ __forceinline__ float4 group_factor(const float* inv, int c, int groups, int size) {
  const int g = min(c / size, groups - 1);
  if (c + 3 < (g + 1) * size || g == groups - 1) return make_float4(inv[g], inv[g], inv[g], inv[g]);
  return make_float4(inv[g], inv[min((c + 1) / size, groups - 1)], inv[min((c + 2) / size, groups - 1)], inv[min((c + 3) / size, groups - 1)]);
}

// CS: CTAs per row; TWO: two normed sources
template <int CS, bool TWO>
__global__ void __launch_bounds__(kThreads) sandwich_kernel(const SandwichParams p) {
  constexpr int NS = TWO ? 2 : 1;
  extern __shared__ __align__(16) float smem[];      // values of the CTA's columns [NS][per], then 4 x groups statistics
  __shared__ float red[kWarps], side_stat[2][2], t_w[NS][kTerms];
  __shared__ long long t_off[NS][kTerms];
  pdl_launch_dependents();
  pdl_wait();
  const int m = blockIdx.x / CS, part = CS > 1 ? blockIdx.x % CS : 0, tid = threadIdx.x;
  const int per = ((p.ld / 4 + CS - 1) / CS) * 4;            // columns per CTA, in fours
  const int c0 = part * per, c1 = min(p.ld, c0 + per);
  float* stat = smem + NS * per;
  float* inv = stat + 2 * p.groups;
#pragma unroll
  for (int s = 0; s < NS; ++s) {
    const B2Source& q = p.src[s];
    for (int t = tid; t < q.slots * q.slices; t += kThreads) {       // where the row's values are and what they count
      const int slot = t / q.slices;
      long long r = q.row_of ? q.row_of[m * q.slots + slot] : (long long)m * q.slots + slot;
      if (p.vocab > 0 && (r < 0 || r >= p.vocab)) {
        if (part == 0 && p.flag) p.flag[0] = 1;
        r = 0;
      }
      t_off[s][t] = r * q.row + (t - slot * q.slices) * q.slice;
      t_w[s][t] = q.slot_w ? q.slot_w[m * q.slots + slot] : 1.f;
    }
  }
  __syncthreads();
  float side[2] = {1.f, 1.f};
#pragma unroll
  for (int s = 0; s < NS; ++s) {
    const B2Source& q = p.src[s];
    const int terms = q.slots * q.slices;
    float ssq = 0.f;
    for (int c = c0 + tid * 4; c < c1; c += kThreads * 4) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int u0 = 0; u0 < terms; u0 += 8) {       // eight values in flight; slots in order, slices of a slot in order
        float4 v[8];
        float wt[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
          wt[u] = 0.f;
          if (u0 + u < terms) {
            v[u] = value4(q, t_off[s][u0 + u] + c);
            wt[u] = t_w[s][u0 + u];
          }
        }
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          a.x = fmaf(wt[u], v[u].x, a.x);
          a.y = fmaf(wt[u], v[u].y, a.y);
          a.z = fmaf(wt[u], v[u].z, a.z);
          a.w = fmaf(wt[u], v[u].w, a.w);
        }
      }
      if (!TWO) a = make_float4(a.x * q.factor, a.y * q.factor, a.z * q.factor, a.w * q.factor);
      *reinterpret_cast<float4*>(smem + s * per + c - c0) = a;
      if (TWO) ssq += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;     // padding columns are zero
    }
    if (TWO) {
      ssq = warp_sum(ssq);
      __syncthreads();
      if ((tid & 31) == 0) red[tid >> 5] = ssq;
      __syncthreads();
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < kWarps; ++i) a += red[i];
      side[s] = a;
    }
  }
  if (TWO) {
    if (CS > 1) {
      cg::cluster_group cl = cg::this_cluster();
      if (tid < 2) side_stat[0][tid] = side[tid];
      cl.sync();
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        side[s] = 0.f;
#pragma unroll
        for (int i = 0; i < CS; ++i) side[s] += *cl.map_shared_rank(&side_stat[0][s], i);
      }
    }
#pragma unroll
    for (int s = 0; s < 2; ++s)
      if (p.src[s].norm) side[s] = p.src[s].factor / sqrtf(side[s] / (float)p.width + p.eps);
      else side[s] = p.src[s].factor;
    for (int c = c0 + tid * 4; c < c1; c += kThreads * 4) {
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        const float4 a = *reinterpret_cast<const float4*>(smem + (NS - 1) * s * per + c - c0);
        const float4 w = p.src[s].norm ? *reinterpret_cast<const float4*>(p.src[s].norm + c) : make_float4(1.f, 1.f, 1.f, 1.f);
        y.x = fmaf(a.x * side[s], w.x, y.x);
        y.y = fmaf(a.y * side[s], w.y, y.y);
        y.z = fmaf(a.z * side[s], w.z, y.z);
        y.w = fmaf(a.w * side[s], w.w, y.w);
      }
      *reinterpret_cast<float4*>(smem + c - c0) = y;
    }
  }
  if (p.post) group_stats<CS>(smem - c0, c0, c1, p.groups, p.size, p.eps, red, stat, inv);
  for (int c = c0 + tid * 4; c < c1; c += kThreads * 4) {
    float4 y = *reinterpret_cast<const float4*>(smem + c - c0);
    if (p.post) {
      const float4 r = group_factor(inv, c, p.groups, p.size), w = *reinterpret_cast<const float4*>(p.post + c);
      y = make_float4(y.x * r.x * w.x, y.y * r.y * w.y, y.z * r.z * w.z, y.w * r.w * w.w);
    }
    if (p.x_in) {
      const float4 x = __ldcg(reinterpret_cast<const float4*>(p.x_in + (size_t)m * p.ld + c));
      y = make_float4(y.x + x.x, y.y + x.y, y.z + x.z, y.w + x.w);
    }
    if (p.x_out) *reinterpret_cast<float4*>(p.x_out + (size_t)m * p.ld + c) = y;
    *reinterpret_cast<float4*>(smem + c - c0) = y;
  }
  group_stats<CS>(smem - c0, c0, c1, p.groups, p.size, p.eps, red, stat + p.groups, inv + p.groups);
  for (int c = c0 + tid * 4; c < c1; c += kThreads * 4) {
    float4 y = *reinterpret_cast<const float4*>(smem + c - c0);
    const float4 r = group_factor(inv + p.groups, c, p.groups, p.size), w = *reinterpret_cast<const float4*>(p.next + c);
    y = make_float4(y.x * r.x * w.x, y.y * r.y * w.y, y.z * r.z * w.z, y.w * r.w * w.w);
    const size_t at = ((size_t)m * p.ld + c) / 4;
    if (p.h_f32) reinterpret_cast<float4*>(p.h)[at] = y;
    else reinterpret_cast<uint2*>(p.h)[at] = make_uint2(pack_bf16(y.x, y.y), pack_bf16(y.z, y.w));
  }
  if (CS > 1) cg::this_cluster().sync();    // no CTA leaves while another may still read its statistics
}

// ------------------------------------------------------------------ groups of whole 128s
constexpr int kRuns = 64;       // runs of 128 columns of a row

// The sum of `per` neighbouring runs from `first`
__device__ __forceinline__ float run_sums(const float* stat, int first, int per) {
  float a = 0.f;
  for (int i = threadIdx.x & 31; i < per; i += 32) a += stat[first + i];
  return warp_sum(a);
}

// NT threads; Q: runs of a warp; TF: values of a column in flight; MB: CTAs per SM
template <bool TWO, int NT, int Q, int TF, int MB>
__global__ void __launch_bounds__(NT, MB) sandwich_runs_kernel(const SandwichParams p) {
  constexpr int NS = TWO ? 2 : 1, NW = NT / 32;
  __shared__ float stat[4][kRuns];           // sums of squares of the runs: of the two results, of y, of x'
  const int m = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int runs = p.ld / 128, group = p.size / 128;      // runs of the row, of a group
  pdl_launch_dependents();
  pdl_wait();
  auto squares = [&](const float4 (&v)[Q], float* to) {
#pragma unroll
    for (int u = 0; u < Q; ++u) {
      const float s = warp_sum(v[u].x * v[u].x + v[u].y * v[u].y + v[u].z * v[u].z + v[u].w * v[u].w);
      if (lane == 0 && u * NW + warp < runs) to[u * NW + warp] = s;
    }
  };
  // 1 / root mean square of the group of every run of this warp
  auto factors = [&](float* of, float (&inv)[Q]) {
    int have = -1;
    float last = 0.f;
#pragma unroll
    for (int u = 0; u < Q; ++u) {
      const int g = min(u * NW + warp, runs - 1) / group;
      if (g != have) last = 1.f / sqrtf(run_sums(of, g * group, group) / (float)p.size + p.eps);
      have = g;
      inv[u] = last;
    }
  };
  float4 y[NS][Q], x[Q];
#pragma unroll
  for (int u = 0; u < Q; ++u) {
    const bool in = u * NW + warp < runs && p.x_in;
    const int c = (u * NW + warp) * 128 + lane * 4;
    x[u] = in ? __ldcg(reinterpret_cast<const float4*>(p.x_in + (size_t)m * p.ld + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int s = 0; s < NS; ++s) {
    const B2Source& q = p.src[s];
    const int terms = q.slots * q.slices;
#pragma unroll
    for (int u = 0; u < Q; ++u) y[s][u] = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int t0 = 0; t0 < terms; t0 += TF) {       // slots in order, slices of a slot in order
      long long off[TF];
      float wt[TF];
#pragma unroll
      for (int i = 0; i < TF; ++i) {
        const int t = min(t0 + i, terms - 1), slot = q.slices > 1 ? t / q.slices : t;
        long long r = q.row_of ? q.row_of[m * q.slots + slot] : (long long)m * q.slots + slot;
        if (p.vocab > 0 && (r < 0 || r >= p.vocab)) {
          if (threadIdx.x == 0 && p.flag) p.flag[0] = 1;
          r = 0;
        }
        off[i] = r * q.row + (t - slot * q.slices) * q.slice;
        wt[i] = t0 + i < terms ? (q.slot_w ? q.slot_w[m * q.slots + slot] : 1.f) : 0.f;
      }
#pragma unroll
      for (int u = 0; u < Q; ++u) {
        if (u * NW + warp >= runs) break;
        const int c = (u * NW + warp) * 128 + lane * 4;
        float4 v[TF];
#pragma unroll
        for (int i = 0; i < TF; ++i) v[i] = t0 + i < terms ? value4(q, off[i] + c) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < TF; ++i) {
          y[s][u].x = fmaf(wt[i], v[i].x, y[s][u].x);
          y[s][u].y = fmaf(wt[i], v[i].y, y[s][u].y);
          y[s][u].z = fmaf(wt[i], v[i].z, y[s][u].z);
          y[s][u].w = fmaf(wt[i], v[i].w, y[s][u].w);
        }
      }
    }
  }
  if (TWO) {
#pragma unroll
    for (int s = 0; s < NS; ++s) squares(y[s], stat[s]);
    __syncthreads();
    float f[NS];
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      f[s] = p.src[s].factor;
      if (p.src[s].norm) f[s] /= sqrtf(run_sums(stat[s], 0, runs) / (float)p.width + p.eps);
    }
#pragma unroll
    for (int u = 0; u < Q; ++u) {
      if (u * NW + warp >= runs) break;
      const int c = (u * NW + warp) * 128 + lane * 4;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int s = 0; s < NS; ++s) {
        const float4 w = p.src[s].norm ? *reinterpret_cast<const float4*>(p.src[s].norm + c) : make_float4(1.f, 1.f, 1.f, 1.f);
        a.x = fmaf(y[s][u].x * f[s], w.x, a.x);
        a.y = fmaf(y[s][u].y * f[s], w.y, a.y);
        a.z = fmaf(y[s][u].z * f[s], w.z, a.z);
        a.w = fmaf(y[s][u].w * f[s], w.w, a.w);
      }
      y[0][u] = a;
    }
  } else {
    const float f = p.src[0].factor;
#pragma unroll
    for (int u = 0; u < Q; ++u) y[0][u] = make_float4(y[0][u].x * f, y[0][u].y * f, y[0][u].z * f, y[0][u].w * f);
  }
  float inv[Q];
  if (p.post) {
    squares(y[0], stat[2]);
    __syncthreads();
    factors(stat[2], inv);
  }
#pragma unroll
  for (int u = 0; u < Q; ++u) {
    if (u * NW + warp >= runs) break;
    const int c = (u * NW + warp) * 128 + lane * 4;
    float4 v = y[0][u];
    if (p.post) {
      const float4 w = *reinterpret_cast<const float4*>(p.post + c);
      v = make_float4(v.x * inv[u] * w.x, v.y * inv[u] * w.y, v.z * inv[u] * w.z, v.w * inv[u] * w.w);
    }
    x[u] = make_float4(v.x + x[u].x, v.y + x[u].y, v.z + x[u].z, v.w + x[u].w);
    if (p.x_out) *reinterpret_cast<float4*>(p.x_out + (size_t)m * p.ld + c) = x[u];
  }
  squares(x, stat[3]);
  __syncthreads();
  factors(stat[3], inv);
#pragma unroll
  for (int u = 0; u < Q; ++u) {
    if (u * NW + warp >= runs) break;
    const int c = (u * NW + warp) * 128 + lane * 4;
    const float4 w = *reinterpret_cast<const float4*>(p.next + c);
    const float4 v = make_float4(x[u].x * inv[u] * w.x, x[u].y * inv[u] * w.y, x[u].z * inv[u] * w.z, x[u].w * inv[u] * w.w);
    const size_t at = ((size_t)m * p.ld + c) / 4;
    if (p.h_f32) reinterpret_cast<float4*>(p.h)[at] = v;
    else reinterpret_cast<uint2*>(p.h)[at] = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
  }
}

int launch_kernel(void (*kernel)(SandwichParams), const SandwichParams& p, int cs, int threads, size_t smem, cudaStream_t st) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.M * cs);
  cfg.blockDim = dim3(threads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = cs;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  static const bool no_pdl = getenv("B2_NO_PDL") != nullptr;  // measurement switch, as in b2_launch
  cfg.numAttrs = no_pdl ? 1 : 2;
  return (int)cudaLaunchKernelEx(&cfg, kernel, p);
}

template <bool TWO>
int launch_runs(const SandwichParams& p, cudaStream_t st) {
  // measured: threads and values in flight that fill the SMs with many rows, and the shortest chain for few
  if (p.M > 64) {
    if (p.ld <= 1024) return launch_kernel(sandwich_runs_kernel<TWO, 128, 2, 2, 8>, p, 1, 128, 0, st);
    if (p.ld <= 2048) return launch_kernel(sandwich_runs_kernel<TWO, 128, 4, 2, 8>, p, 1, 128, 0, st);
    if (p.ld <= 4096) return launch_kernel(sandwich_runs_kernel<TWO, 256, 4, 4, 4>, p, 1, 256, 0, st);
    return launch_kernel(sandwich_runs_kernel<TWO, 256, 8, 4, 1>, p, 1, 256, 0, st);
  }
  if (p.ld <= 1024) return launch_kernel(sandwich_runs_kernel<TWO, 256, 1, 4, 4>, p, 1, 256, 0, st);
  if (p.ld <= 2048) return launch_kernel(sandwich_runs_kernel<TWO, 512, 1, 4, 2>, p, 1, 512, 0, st);
  if (p.ld <= 4096) return launch_kernel(sandwich_runs_kernel<TWO, 1024, 1, 4, 1>, p, 1, 1024, 0, st);
  return launch_kernel(sandwich_runs_kernel<TWO, 1024, 2, 4, 1>, p, 1, 1024, 0, st);
}

template <int CS, bool TWO>
int launch_form(const SandwichParams& p, cudaStream_t st) {
  if (p.width == p.ld && p.size % 128 == 0 && p.ld <= 128 * kRuns) return launch_runs<TWO>(p, st);
  const int per = ((p.ld / 4 + CS - 1) / CS) * 4;
  const size_t smem = ((size_t)(TWO ? 2 : 1) * per + 4 * p.groups) * sizeof(float);
  if (smem > 200 * 1024) return -5;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(sandwich_kernel<CS, TWO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return launch_kernel(sandwich_kernel<CS, TWO>, p, CS, kThreads, smem, st);
}

template <int CS>
int launch(const SandwichParams& p, cudaStream_t st) {
  return p.n_src == 2 ? launch_form<CS, true>(p, st) : launch_form<CS, false>(p, st);
}

}  // namespace

// src: one or two sources (two: each with a norm or without); see SandwichParams.  x_in and x_out may be the same buffer.
extern "C" int b2_sandwich(const B2Source* src, int n_src, int vocab, int* flag, int M, int width, int ld, int groups, float eps,
                           const float* post, const float* next, const float* x_in, float* x_out, void* h, int h_f32, void* stream) {
  if (M < 1 || ld % 4 || width > ld || groups < 1 || groups > kGroups || width % groups || n_src < 1 || n_src > 2 || !next || !h) return -1;
  SandwichParams p = {};
  for (int s = 0; s < n_src; ++s) {
    const B2Source& q = src[s];
    if (!q.y || q.slots < 1 || q.slices < 1 || q.slots * q.slices > kTerms || q.row % 4 || q.slice % 4) return -2;
    if (n_src == 1 && q.norm) return -3;
    p.src[s] = q;
  }
  if (vocab > 0 && (n_src != 1 || !src[0].row_of)) return -4;
  p.n_src = n_src; p.vocab = vocab; p.flag = flag; p.M = M; p.width = width; p.ld = ld; p.groups = groups; p.size = width / groups;
  p.eps = eps; p.post = post; p.next = next; p.x_in = x_in; p.x_out = x_out; p.h = h; p.h_f32 = h_f32;
  cudaStream_t st = (cudaStream_t)stream;
  // as in the other boundary kernels, the split over CTAs depends on the width alone up to the row count where whole rows fill
  // the GPU
  if (M > 64 || ld < 1024) return launch<1>(p, st);
  return ld < 4096 ? launch<4>(p, st) : launch<8>(p, st);
}

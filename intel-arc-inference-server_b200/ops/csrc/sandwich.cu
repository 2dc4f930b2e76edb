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
// A row is handled by one CTA, or by a cluster of up to 8 CTAs that share the columns and exchange their sums of squares through
// distributed shared memory (few rows).
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

template <int CS, bool TWO>
int launch_form(const SandwichParams& p, cudaStream_t st) {
  const int per = ((p.ld / 4 + CS - 1) / CS) * 4;
  const size_t smem = ((size_t)(TWO ? 2 : 1) * per + 4 * p.groups) * sizeof(float);
  if (smem > 200 * 1024) return -5;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(sandwich_kernel<CS, TWO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(p.M * CS);
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = CS;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  static const bool no_pdl = getenv("B2_NO_PDL") != nullptr;  // measurement switch, as in b2_launch
  cfg.numAttrs = no_pdl ? 1 : 2;
  return (int)cudaLaunchKernelEx(&cfg, sandwich_kernel<CS, TWO>, p);
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

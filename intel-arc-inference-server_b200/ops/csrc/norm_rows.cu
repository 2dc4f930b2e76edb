// Layer norm on fp32 residual rows.
//
//   sublayer_norm_kernel   x += LN(y) * w, h = x rounded for the next sublayer.  y is what a sublayer left: split-K slices
//                          of a linear, or a mixture-of-experts row's weighted slots (slices per slot, or rows of the
//                          expert-sorted buffer).  The fold, the statistics and the residual sum are fp32; the variance is
//                          taken from the deviations.  With `add` 0 the norm is the row's own (no residual), with `w`
//                          null the sum itself is added without a norm.
//   layer_norm_rows_kernel LN of selected residual rows (the model's output norm)
//   embed_rows_kernel      residual rows = embedding rows of the step's tokens
//
// A row is handled by one CTA, or by a cluster of up to 8 CTAs that share the columns and exchange the two statistics
// through distributed shared memory (few rows: the loads of one row then come from several SMs).
#include "common.cuh"

#include <cooperative_groups.h>

using namespace b2;
namespace cg = cooperative_groups;

namespace {

constexpr int kThreads = 256;
constexpr int kTerms = 256;     // slots x slices of a row

struct SubNormParams {
  const void* y;             // fp32 (or bf16 with y_bf16) values
  const int* row_of;         // slot form over sorted rows: row of (m, slot); null: slot rows are m * slots + slot
  const float* slot_w;       // [M][slots]; null: every slot counts once
  long long slice;           // elements between split-K slices of a value row
  long long row;             // elements between value rows
  int slots, slices, y_bf16;
  int M, width, ld;          // true columns; columns of x / h rows (the rest is padding, kept zero)
  const float* w;            // [width]
  float eps;
  float* x;                  // [M][ld] fp32, in place
  void* h;                   // [M][ld] bf16 or fp32
  int h_f32, add;
};

__device__ __forceinline__ void store_h(void* h, int f32, size_t i, float v) {
  if (f32) reinterpret_cast<float*>(h)[i] = v;
  else reinterpret_cast<__nv_bfloat16*>(h)[i] = __float2bfloat16(v);
}

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) s += red[i];
  return s;
}

// CS: CTAs per row (cluster size); columns of the row's part live in shared memory between the passes
template <int CS>
__global__ void __launch_bounds__(kThreads) sublayer_norm_kernel(const SubNormParams p) {
  extern __shared__ __align__(16) float vals[];
  __shared__ float red[kThreads / 32], stat[2], t_w[kTerms];
  __shared__ long long t_off[kTerms];
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x / CS, part = CS > 1 ? blockIdx.x % CS : 0;
  const int per = ((p.ld / 4 + CS - 1) / CS) * 4;            // columns per CTA, in fours
  const int c0 = part * per, c1 = min(p.ld, c0 + per);
  const int terms = p.slots * p.slices;
  for (int t = threadIdx.x; t < terms; t += kThreads) {       // where the row's values are and what they count
    const int s = t / p.slices, q = t - s * p.slices;
    const long long r = p.row_of ? p.row_of[m * p.slots + s] : (long long)m * p.slots + s;
    t_off[t] = r * p.row + q * p.slice;
    t_w[t] = p.slot_w ? p.slot_w[m * p.slots + s] : 1.f;
  }
  __syncthreads();
  float sum = 0.f;
  for (int c = c0 + threadIdx.x * 4; c < c1; c += kThreads * 4) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int u0 = 0; u0 < terms; u0 += 8) {       // eight values in flight; slots in order, slices of a slot in order
      float4 v[8];
      float wt[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const int t = u0 + u;
        v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        wt[u] = 0.f;
        if (t < terms) {
          const long long off = t_off[t] + c;
          wt[u] = t_w[t];
          if (p.y_bf16) {
            const uint2 raw = __ldcg(reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p.y) + off));
            v[u] = make_float4(bf16_lo(raw.x), bf16_hi(raw.x), bf16_lo(raw.y), bf16_hi(raw.y));
          } else {
            v[u] = __ldcg(reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p.y) + off));
          }
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
    float e[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (c + j < p.width) sum += e[j];
    }
    *reinterpret_cast<float4*>(vals + c - c0) = a;
  }
  float mean = 0.f, rstd = 1.f;
  if (p.w) {
    sum = block_sum(sum, red);
    if (CS > 1) {
      cg::cluster_group cl = cg::this_cluster();
      if (threadIdx.x == 0) stat[0] = sum;
      cl.sync();
      sum = 0.f;
#pragma unroll
      for (int i = 0; i < CS; ++i) sum += *cl.map_shared_rank(&stat[0], i);
    }
    mean = sum / (float)p.width;
    float dev = 0.f;
    for (int c = c0 + threadIdx.x * 4; c < c1; c += kThreads * 4)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j < p.width) {
          const float d = vals[c - c0 + j] - mean;
          dev = fmaf(d, d, dev);
        }
    dev = block_sum(dev, red);
    if (CS > 1) {
      cg::cluster_group cl = cg::this_cluster();
      if (threadIdx.x == 0) stat[1] = dev;
      cl.sync();
      dev = 0.f;
#pragma unroll
      for (int i = 0; i < CS; ++i) dev += *cl.map_shared_rank(&stat[1], i);
    }
    rstd = 1.f / sqrtf(dev / (float)p.width + p.eps);
  }
  for (int c = c0 + threadIdx.x * 4; c < c1; c += kThreads * 4) {
    float4* xr = reinterpret_cast<float4*>(p.x + (size_t)m * p.ld + c);
    float4 xv = p.add ? *xr : make_float4(0.f, 0.f, 0.f, 0.f);
    float e[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (c + j < p.width) e[j] += p.w ? (vals[c - c0 + j] - mean) * rstd * p.w[c + j] : vals[c - c0 + j];
      else e[j] = 0.f;
    }
    if (p.h_f32) reinterpret_cast<float4*>(p.h)[((size_t)m * p.ld + c) / 4] = make_float4(e[0], e[1], e[2], e[3]);
    else reinterpret_cast<uint2*>(p.h)[((size_t)m * p.ld + c) / 4] = make_uint2(pack_bf16(e[0], e[1]), pack_bf16(e[2], e[3]));
    *xr = make_float4(e[0], e[1], e[2], e[3]);
  }
  if (CS > 1) cg::this_cluster().sync();    // no CTA leaves while another may still read its statistics
}

__global__ void __launch_bounds__(kThreads) layer_norm_rows_kernel(const float* __restrict__ x, const int* __restrict__ rows,
                                                                   const float* __restrict__ w, float eps, int width, int ld,
                                                                   void* __restrict__ h, int h_f32) {
  __shared__ float red[kThreads / 32];
  pdl_wait();
  pdl_launch_dependents();
  const float* xr = x + (size_t)(rows ? rows[blockIdx.x] : blockIdx.x) * ld;
  float s = 0.f;
  for (int c = threadIdx.x; c < width; c += kThreads) s += xr[c];
  const float mean = block_sum(s, red) / (float)width;
  float d2 = 0.f;
  for (int c = threadIdx.x; c < width; c += kThreads) {
    const float d = xr[c] - mean;
    d2 = fmaf(d, d, d2);
  }
  const float rstd = 1.f / sqrtf(block_sum(d2, red) / (float)width + eps);
  for (int c = threadIdx.x; c < ld; c += kThreads)
    store_h(h, h_f32, (size_t)blockIdx.x * ld + c, c < width ? (xr[c] - mean) * rstd * w[c] : 0.f);
}

// tokens outside the vocabulary set the flag and read row 0
__global__ void __launch_bounds__(kThreads) embed_rows_kernel(const void* __restrict__ embed, const int* __restrict__ tokens,
                                                              int vocab, int ld, float* __restrict__ x, void* __restrict__ h,
                                                              int f32, int* __restrict__ flag) {
  pdl_wait();
  pdl_launch_dependents();
  int tok = tokens[blockIdx.x];
  if (tok < 0 || tok >= vocab) {
    if (threadIdx.x == 0 && flag) flag[0] = 1;
    tok = 0;
  }
  for (int c = threadIdx.x; c < ld; c += kThreads) {
    const size_t i = (size_t)tok * ld + c, o = (size_t)blockIdx.x * ld + c;
    const float v = f32 ? reinterpret_cast<const float*>(embed)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(embed)[i]);
    x[o] = v;
    store_h(h, f32, o, v);
  }
}

// arg-max of fp32 logit rows as one (value, id) candidate per row; ties go to the lower id
__global__ void __launch_bounds__(kThreads) row_argmax_kernel(const float* __restrict__ logits, int n, float* __restrict__ val,
                                                              int* __restrict__ idx) {
  __shared__ float sv[kThreads];
  __shared__ int si[kThreads];
  pdl_wait();
  pdl_launch_dependents();
  const float* r = logits + (size_t)blockIdx.x * n;
  float b = -INFINITY;
  int bi = 0x7fffffff;
  for (int i = threadIdx.x; i < n; i += kThreads)
    if (r[i] > b) { b = r[i]; bi = i; }
  sv[threadIdx.x] = b;
  si[threadIdx.x] = bi;
  __syncthreads();
  for (int o = kThreads / 2; o > 0; o >>= 1) {
    if (threadIdx.x < o && (sv[threadIdx.x + o] > sv[threadIdx.x] ||
                            (sv[threadIdx.x + o] == sv[threadIdx.x] && si[threadIdx.x + o] < si[threadIdx.x]))) {
      sv[threadIdx.x] = sv[threadIdx.x + o];
      si[threadIdx.x] = si[threadIdx.x + o];
    }
    __syncthreads();
  }
  if (threadIdx.x == 0) { val[blockIdx.x] = sv[0]; idx[blockIdx.x] = si[0]; }
}

template <int CS>
int launch_subnorm(const SubNormParams& p, cudaStream_t st) {
  const size_t smem = (size_t)(((p.ld / 4 + CS - 1) / CS) * 4) * sizeof(float);
  if (smem > 48 * 1024) return -5;
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
  return (int)cudaLaunchKernelEx(&cfg, sublayer_norm_kernel<CS>, p);
}

}  // namespace

extern "C" int b2_sublayer_norm(const void* y, int y_bf16, const int* row_of, const float* slot_w, long long slice,
                                long long row, int slots, int slices, int M, int width, int ld, const float* w, float eps,
                                float* x, void* h, int h_f32, int add, void* stream) {
  if (M < 1 || slots < 1 || slices < 1 || slots * slices > kTerms || ld % 4 || width > ld || row % 4 || slice % 4) return -1;
  SubNormParams p{y, row_of, slot_w, slice, row, slots, slices, y_bf16, M, width, ld, w, eps, x, h, h_f32, add};
  cudaStream_t st = (cudaStream_t)stream;
  // the split over CTAs changes the order of the statistics' sums, so it depends on the width alone up to the row
  // count where whole rows fill the GPU
  if (M > 64 || ld < 1024) return launch_subnorm<1>(p, st);
  return ld < 4096 ? launch_subnorm<4>(p, st) : launch_subnorm<8>(p, st);
}

extern "C" int b2_layer_norm_rows(const float* x, const int* rows, const float* w, float eps, int M, int width, int ld, void* h,
                                  int h_f32, void* stream) {
  if (M < 1 || width > ld) return -1;
  return b2_launch(layer_norm_rows_kernel, dim3(M), dim3(kThreads), 0, (cudaStream_t)stream, true, x, rows, w, eps, width, ld,
                   h, h_f32);
}

extern "C" int b2_embed_rows(const void* embed, const int* tokens, int vocab, int M, int ld, float* x, void* h, int f32,
                             int* flag, void* stream) {
  if (M < 1) return -1;
  return b2_launch(embed_rows_kernel, dim3(M), dim3(kThreads), 0, (cudaStream_t)stream, true, embed, tokens, vocab, ld, x, h,
                   f32, flag);
}

extern "C" int b2_row_argmax(const float* logits, int M, int n, float* val, int* idx, void* stream) {
  if (M < 1 || n < 1) return -1;
  return b2_launch(row_argmax_kernel, dim3(M), dim3(kThreads), 0, (cudaStream_t)stream, true, logits, n, val, idx);
}

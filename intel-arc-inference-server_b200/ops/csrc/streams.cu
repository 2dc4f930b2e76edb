// Residual of several streams (hyper-connections) around a sublayer, in one pass over the rows:
//
//   x'_t = sum_s mix[s][t] x_s + mult out[t] (scale o y)         streams after the sublayer whose result is y
//   u    = sum_t in[t] x'_t,  h = u / sqrt(mean(u^2) + eps) g     what the next sublayer reads (g: one number)
//   h   <- h + (h_before - h) o mu                                optional token shift; h_before: the row before, unshifted
//
// y is what a linear left (split-K slices, folded here, plus its bias); everything is fp32, h is rounded at the end.  The
// first call of a step has no y: all streams start as the embedding row plus a sinusoidal position vector.
//
// Options: a plain residual (no mix, in, out: one stream, x' = x + y); a norm with a factor per column; what comes before a
// pass over a range of layers (the embedding row once more, a vector); several shifted results of one row at a time, each
// with its own mu (a plane of h each).
//
// The streams are read from one buffer and written to another, because a row whose predecessor is in the same step
// computes the predecessor's h again when it belongs to another CTA (a CTA walks `rows_per` rows and keeps the last h).
// The h a sequence starts the next step with goes through `next` [slot]: a step's last row of a sequence leaves it there,
// and the call that adds this mixer's result puts it into the layer's own state (`commit`); no CTA of the call that
// reads a layer's state writes it.
//
// Few rows: a row is shared by a cluster of up to 8 CTAs that exchange the sum of squares through distributed shared
// memory.
#include "common.cuh"

#include <cooperative_groups.h>

using namespace b2;
namespace cg = cooperative_groups;

namespace {

constexpr int kThreads = 256;

struct StreamParams {
  const float* y;            // [slices][M][ld]; null: embedding form
  long long slice;
  int slices;
  const void* embed;         // [vocab][ld]
  const int* tokens;
  const double* freq;        // [width / 2] angle per position; null: no position vector
  int vocab, embed_f32;
  int* flag;                 // set when a token is outside the vocabulary (it reads row 0)
  const int *req, *pos;
  int M, width, ld, rows_per;
  const float* x_in;         // [M][S][ld]
  float* x_out;              // [M][S][ld], or null
  const float *mix, *out;    // [S][S] from, to; [S]
  const float* scale;        // [ld] layer scale, or null
  float mult;
  const float* in;           // [S], null: the plain sum
  const float* g;            // [1], or [ld] with g_cols
  int g_cols;
  const float* bias;         // [ld] of the linear that left y, or null
  const float* add;          // [ld] added to the streams, or null
  int again;                 // the embedding row is added to the streams
  float eps;
  void* h;                   // [M][ld]
  int h_f32;
  const float* mu;           // [planes][ld], null: no shift
  int planes;                // h is [planes][M][ld]
  const float* prev;         // [slots][ld] state of the layer that reads h
  float* next;               // [slots][ld]
  float* commit;             // [slots][ld] state of the layer whose mixer made y, or null
};

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

__device__ __forceinline__ float4 fma4(float a, const float4& x, const float4& y) {
  return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}

// columns c .. c + 3 of a token's embedding with its position vector; the angle is reduced in double
__device__ __forceinline__ float4 embedded(const StreamParams& p, int tok, int pos, int c) {
  float4 v;
  if (p.embed_f32) {
    v = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p.embed) + (size_t)tok * p.ld + c);
  } else {
    const uint2 r = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p.embed) + (size_t)tok * p.ld + c);
    v = make_float4(bf16_lo(r.x), bf16_hi(r.x), bf16_lo(r.y), bf16_hi(r.y));
  }
  if (p.freq) {
    float* e = &v.x;
#pragma unroll
    for (int j = 0; j < 4; j += 2)
      if (c + j < p.width) {
        constexpr double kTurn = 6.283185307179586476925;
        const double a = (double)pos * p.freq[(c + j) >> 1];
        const float r = (float)(a - kTurn * rint(a / kTurn));
        e[j] += sinf(r);
        if (c + j + 1 < p.width) e[j + 1] += cosf(r);
      }
  }
  return v;
}

// EXT: the options at the end of the list above
template <int S, int CS, bool EXT>
__global__ void __launch_bounds__(kThreads) streams_kernel(const StreamParams p) {
  extern __shared__ __align__(16) float vals[];            // u of the row at hand, then h of the row before
  __shared__ float red[kThreads / 32], stat, s_mix[S * S], s_out[S], s_in[S];
  const int tid = threadIdx.x;
  if (tid < S) {
    s_out[tid] = p.y ? (p.out ? p.out[tid] : 1.f) * p.mult : 0.f;
    s_in[tid] = p.in ? p.in[tid] : 1.f;
  }
  if (tid < S * S) s_mix[tid] = !p.y ? 0.f : p.mix ? p.mix[tid] : tid % (S + 1) == 0 ? 1.f : 0.f;
  const float g = EXT && p.g_cols ? 1.f : p.g[0];
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();
  const int part = CS > 1 ? blockIdx.x % CS : 0;
  const int per = ((p.ld / 4 + CS - 1) / CS) * 4;           // columns per CTA, in fours
  const int c0 = part * per, c1 = min(p.ld, c0 + per);
  float* u = vals - c0;
  float* before = vals + per - c0;
  const int r0 = (blockIdx.x / CS) * p.rows_per, r1 = min(p.M, r0 + p.rows_per);

  // u of row m into shared memory (this thread reads back its own columns only); returns the factor that makes it h
  auto pass = [&](int m, bool store) -> float {
    float ssq = 0.f;
    int tok = 0, pos = 0;
    if (!p.y || (EXT && p.again)) {
      tok = p.tokens[m];
      pos = p.pos[m];
      if (tok < 0 || tok >= p.vocab) {
        if (tid == 0 && p.flag) p.flag[0] = 1;
        tok = 0;
      }
    }
    for (int c = c0 + tid * 4; c < c1; c += kThreads * 4) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      if (p.y) {
        float4 x[S], b[8];
#pragma unroll
        for (int s = 0; s < S; ++s) x[s] = __ldcg(reinterpret_cast<const float4*>(p.x_in + ((size_t)m * S + s) * p.ld + c));
#pragma unroll
        for (int s = 0; s < 8; ++s)           // slices <= 8
          b[s] = s < p.slices ? __ldcg(reinterpret_cast<const float4*>(p.y + s * p.slice + (size_t)m * p.ld + c)) : a;
        float4 y = b[0];
#pragma unroll
        for (int s = 1; s < 8; ++s) y = fma4(1.f, b[s], y);
        if (EXT && p.bias) y = fma4(1.f, *reinterpret_cast<const float4*>(p.bias + c), y);
        if (p.scale) {
          const float4 w = *reinterpret_cast<const float4*>(p.scale + c);
          y.x *= w.x; y.y *= w.y; y.z *= w.z; y.w *= w.w;
        }
        float4 ahead = make_float4(0.f, 0.f, 0.f, 0.f);
        if (EXT && p.again) ahead = embedded(p, tok, pos, c);
        if (EXT && p.add) ahead = fma4(1.f, *reinterpret_cast<const float4*>(p.add + c), ahead);
#pragma unroll
        for (int t = 0; t < S; ++t) {
          float4 v = make_float4(s_out[t] * y.x, s_out[t] * y.y, s_out[t] * y.z, s_out[t] * y.w);
#pragma unroll
          for (int s = 0; s < S; ++s) v = fma4(s_mix[s * S + t], x[s], v);
          if (EXT) v = fma4(1.f, ahead, v);
          if (store && p.x_out) *reinterpret_cast<float4*>(p.x_out + ((size_t)m * S + t) * p.ld + c) = v;
          a = fma4(s_in[t], v, a);
        }
      } else {
        float4 v = embedded(p, tok, pos, c);
        if (EXT && p.add) v = fma4(1.f, *reinterpret_cast<const float4*>(p.add + c), v);
#pragma unroll
        for (int t = 0; t < S; ++t) {
          if (store && p.x_out) *reinterpret_cast<float4*>(p.x_out + ((size_t)m * S + t) * p.ld + c) = v;
          a = fma4(s_in[t], v, a);
        }
      }
      ssq += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;     // padding columns are zero
      *reinterpret_cast<float4*>(u + c) = a;
    }
    ssq = block_sum(ssq, red);
    if (CS > 1) {
      cg::cluster_group cl = cg::this_cluster();
      if (tid == 0) stat = ssq;
      cl.sync();
      ssq = 0.f;
#pragma unroll
      for (int i = 0; i < CS; ++i) ssq += *cl.map_shared_rank(&stat, i);
      cl.sync();        // the next pass may write its sum, and no CTA leaves while another may still read
    }
    return g / sqrtf(ssq / (float)p.width + p.eps);
  };

  int have = -1;          // row whose h is in `before`
  for (int m = r0; m < r1; ++m) {
    const int req = p.req[m];
    bool follows = false;
    if (p.mu) {
      follows = m > 0 && p.req[m - 1] == req;
      if (follows && have != m - 1) {
        const float r = pass(m - 1, false);
        for (int c = c0 + tid * 4; c < c1; c += kThreads * 4)
#pragma unroll
          for (int j = 0; j < 4; ++j) before[c + j] = u[c + j] * r * (EXT && p.g_cols ? p.g[c + j] : 1.f);
      }
    }
    const bool last = m + 1 == p.M || p.req[m + 1] != req;
    const bool first = p.mu && p.pos[m] == 0;
    const float r = pass(m, true);
    for (int c = c0 + tid * 4; c < c1; c += kThreads * 4) {
      const size_t st = (size_t)req * p.ld + c;
      if (p.commit && last) *reinterpret_cast<float4*>(p.commit + st) = __ldcg(reinterpret_cast<const float4*>(p.next + st));
      float4 h = *reinterpret_cast<const float4*>(u + c);
      h.x *= r; h.y *= r; h.z *= r; h.w *= r;
      if (EXT && p.g_cols) {
        const float4 w = *reinterpret_cast<const float4*>(p.g + c);
        h.x *= w.x; h.y *= w.y; h.z *= w.z; h.w *= w.w;
      }
      auto store = [&](int plane, const float4& o) {
        const size_t at = (((size_t)plane * p.M + m) * p.ld + c) / 4;
        if (p.h_f32) reinterpret_cast<float4*>(p.h)[at] = o;
        else reinterpret_cast<uint2*>(p.h)[at] = make_uint2(pack_bf16(o.x, o.y), pack_bf16(o.z, o.w));
      };
      if (p.mu) {
        float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
        if (follows) b = *reinterpret_cast<const float4*>(before + c);
        else if (!first) b = __ldcg(reinterpret_cast<const float4*>(p.prev + st));
        for (int i = 0; i < (EXT ? p.planes : 1); ++i) {
          const float4 w = *reinterpret_cast<const float4*>(p.mu + (size_t)i * p.ld + c);
          store(i, make_float4(fmaf(b.x - h.x, w.x, h.x), fmaf(b.y - h.y, w.y, h.y), fmaf(b.z - h.z, w.z, h.z), fmaf(b.w - h.w, w.w, h.w)));
        }
        *reinterpret_cast<float4*>(before + c) = h;
        if (last) *reinterpret_cast<float4*>(p.next + st) = h;
      } else {
        store(0, h);
      }
    }
    have = m;
  }
}

template <int S, int CS, bool EXT>
int launch_form(const StreamParams& p, cudaStream_t st) {
  const size_t smem = 2 * (size_t)(((p.ld / 4 + CS - 1) / CS) * 4) * sizeof(float);
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) return -5;
    cudaError_t e = cudaFuncSetAttribute(streams_kernel<S, CS, EXT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(((p.M + p.rows_per - 1) / p.rows_per) * CS);
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
  return (int)cudaLaunchKernelEx(&cfg, streams_kernel<S, CS, EXT>, p);
}

template <int S, int CS>
int launch(const StreamParams& p, cudaStream_t st) {
  return p.g_cols || p.bias || p.add || p.again || p.planes > 1 ? launch_form<S, CS, true>(p, st) : launch_form<S, CS, false>(p, st);
}

template <int S>
int launch_streams(StreamParams& p, cudaStream_t st) {
  // rows spread over clusters while they are few; many rows with a shift are walked, one row computed twice per CTA
  if (p.M > 64) {
    p.rows_per = p.mu ? (p.M + 148 * 4 - 1) / (148 * 4) : 1;
    return launch<S, 1>(p, st);
  }
  p.rows_per = 1;
  if (p.ld < 1024) return launch<S, 1>(p, st);
  return p.ld < 4096 ? launch<S, 4>(p, st) : launch<S, 8>(p, st);
}

}  // namespace

// y null: the embedding form (embed .. flag).  See StreamParams for the rest; rows of a sequence are consecutive.
extern "C" int b2_streams(const float* y, long long slice, int slices, const void* embed, const int* tokens, const double* freq,
                          int vocab, int embed_f32, int* flag, const int* req, const int* pos, int M, int streams, int width,
                          int ld, const float* x_in, float* x_out, const float* mix, const float* out, const float* scale,
                          float mult, const float* in, const float* g, int g_cols, float eps, void* h, int h_f32, const float* mu,
                          int planes, const float* prev, float* next, float* commit, const float* bias, const float* add, int again,
                          void* stream) {
  if (M < 1 || ld % 4 || width > ld || slice % 4 || (y && (slices < 1 || slices > 8 || !x_in)) || (!y && !embed)) return -1;
  if ((mu && (!prev || !next || planes < 1)) || (commit && !next) || (again && (!embed || !tokens))) return -2;
  if (y && streams > 1 && (!mix || !out)) return -4;
  StreamParams p{y, slice, slices, embed, tokens, freq, vocab, embed_f32, flag, req, pos, M, width, ld, 1, x_in, x_out, mix,
                 out, scale, mult, in, g, g_cols, bias, add, again, eps, h, h_f32, mu, planes, prev, next, commit};
  cudaStream_t st = (cudaStream_t)stream;
  switch (streams) {
    case 1: return launch_streams<1>(p, st);
    case 2: return launch_streams<2>(p, st);
    case 3: return launch_streams<3>(p, st);
    case 4: return launch_streams<4>(p, st);
    case 5: return launch_streams<5>(p, st);
    case 6: return launch_streams<6>(p, st);
    case 7: return launch_streams<7>(p, st);
    case 8: return launch_streams<8>(p, st);
  }
  return -3;
}

// Gated recurrence whose gates read the current token only (minGRU), element by element:
//
//   z = sigmoid(a),  c = u + 1/2 where u >= 0, sigmoid(u) where u < 0,  S <- (1 - z) S + z c,  out = mult S silu(g)
//
// a, u, g are columns of a projection (fp32 slices); everything is fp32, out is rounded at the end.
//
//   mingru_rows_kernel      rows in order, a thread per column and sequence
//   mingru_segments_kernel  prompt segments: a CTA walks 32 columns in blocks of rows; its warps take parts of a block, which
//                           they first reduce to S_out = A S_in + B, then meet in shared memory
//
// A sequence's first row (position 0) starts from zeros whatever its slot holds.
#include "common.cuh"

using namespace b2;

namespace {

__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

struct GruParams {
  const float* part;       // [slices][M][N]; columns col: a [W] | u [W] | g [W]
  int slices, M, N, col, W;
  const float *bias_a, *bias_u;    // [W]
  const int *req, *pos;
  const int* segs;         // segments form: [n][4]: first row, rows, slot (rows counted from row0)
  int row0;
  float mult;
  float* state;            // [slots][W]
  void* out;               // [M][ldo]
  int ldo;
};

// 1 - z, and z c; FAST: the intrinsics of models served in bf16
template <bool FAST>
__device__ __forceinline__ float exp_f(float x) { return FAST ? __expf(x) : expf(x); }
template <bool FAST>
__device__ __forceinline__ float div_f(float x, float y) { return FAST ? __fdividef(x, y) : x / y; }
template <bool FAST>
__device__ __forceinline__ float2 gates(float a, float u) {
  const float e = exp_f<FAST>(-fabsf(a)), big = div_f<FAST>(1.f, 1.f + e), small = e * big;      // sigmoid(|a|), sigmoid(-|a|)
  const float z = a >= 0.f ? big : small, keep = a >= 0.f ? small : big;
  const float c = u >= 0.f ? u + 0.5f : div_f<FAST>(1.f, 1.f + exp_f<FAST>(fminf(-u, 80.f)));
  return make_float2(keep, z * c);
}
template <bool FAST>
__device__ __forceinline__ float silu_f(float x) { return div_f<FAST>(x, 1.f + exp_f<FAST>(fminf(-x, 80.f))); }

template <typename T>
__global__ void __launch_bounds__(128) mingru_rows_kernel(const GruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = blockIdx.x * 128 + threadIdx.x, first = blockIdx.y;
  const int slot = p.req[first];
  if (c >= p.W || (first > 0 && p.req[first - 1] == slot)) return;
  float* st = p.state + (size_t)slot * p.W + c;
  float s = p.pos[first] == 0 ? 0.f : __ldcg(st);
  const float ba = p.bias_a[c], bu = p.bias_u[c];
  const size_t slice = (size_t)p.M * p.N;
  for (int m = first; m < p.row0 && p.req[m] == slot; ++m) {
    const float* x = p.part + (size_t)m * p.N + p.col + c;
    float v[3][8];
#pragma unroll
    for (int q = 0; q < 8; ++q)
#pragma unroll
      for (int i = 0; i < 3; ++i) v[i][q] = q < p.slices ? __ldcg(x + q * slice + i * p.W) : 0.f;
    float a = 0.f, u = 0.f, g = 0.f;
#pragma unroll
    for (int q = 0; q < 8; ++q) { a += v[0][q]; u += v[1][q]; g += v[2][q]; }
    const float2 k = gates<sizeof(T) == 2>(a + ba, u + bu);
    s = fmaf(k.x, s, k.y);
    put(reinterpret_cast<T*>(p.out) + (size_t)m * p.ldo + c, p.mult * s * silu_f<sizeof(T) == 2>(g));
  }
  *st = s;
}

constexpr int kParts = 16, kRows = 8;      // warps, rows of a warp's part

template <typename T>
__global__ void __launch_bounds__(kParts * 32) mingru_segments_kernel(const GruParams p) {
  __shared__ float2 s_ab[2][kParts][32];
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c = blockIdx.x * 32 + lane;
  const int* seg = p.segs + blockIdx.y * 4;
  const int row0 = p.row0 + seg[0], rows = seg[1], slot = seg[2];
  float* st = p.state + (size_t)slot * p.W + c;
  float s = p.pos[row0] == 0 ? 0.f : __ldcg(st);
  const float ba = p.bias_a[c], bu = p.bias_u[c];
  const float* x = p.part + (size_t)row0 * p.N + p.col + c;
  T* out = reinterpret_cast<T*>(p.out) + (size_t)row0 * p.ldo + c;
  const int blocks = (rows + kParts * kRows - 1) / (kParts * kRows);
  float a[kRows], u[kRows], g[kRows];
  auto load = [&](int b) {
    const int r0 = (b * kParts + warp) * kRows;
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const bool ok = r0 + i < rows;
      const float* y = x + (size_t)(r0 + i) * p.N;
      a[i] = ok ? __ldcg(y) : 0.f;
      u[i] = ok ? __ldcg(y + p.W) : 0.f;
      g[i] = ok ? __ldcg(y + 2 * p.W) : 0.f;
    }
  };
  load(0);
  for (int b = 0; b < blocks; ++b) {
    const int r0 = (b * kParts + warp) * kRows;
    float2 k[kRows], ab = make_float2(1.f, 0.f);
    float gate[kRows];
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      k[i] = r0 + i < rows ? gates<sizeof(T) == 2>(a[i] + ba, u[i] + bu) : make_float2(1.f, 0.f);      // rows past the end keep the state
      gate[i] = p.mult * silu_f<sizeof(T) == 2>(g[i]);
      ab = make_float2(ab.x * k[i].x, fmaf(k[i].x, ab.y, k[i].y));
    }
    if (b + 1 < blocks) load(b + 1);
    s_ab[b & 1][warp][lane] = ab;
    __syncthreads();
    float cur = s;
#pragma unroll
    for (int w = 0; w < kParts; ++w) {
      const float2 v = s_ab[b & 1][w][lane];
      if (w == warp) cur = s;
      s = fmaf(v.x, s, v.y);
    }
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      cur = fmaf(k[i].x, cur, k[i].y);
      if (r0 + i < rows) put(out + (size_t)(r0 + i) * p.ldo, cur * gate[i]);
    }
  }
  __syncthreads();
  if (warp == 0) *st = s;
}

}  // namespace

// Rows 0 .. n1 - 1 one by one (a sequence per run of equal `req`), then n_segs segments over the rows from n1 on (segs: 4 ints
// each: first row counted from n1, rows, slot, unused).  W is a multiple of 32.
extern "C" int b2_mingru(const float* part, int slices, int M, int N, int col, int W, const float* bias_a, const float* bias_u,
                         const int* req, const int* pos, int n1, const int* segs, int n_segs, float mult, float* state, void* out,
                         int ldo, int f32, void* stream) {
  if (M < 1 || slices < 1 || slices > 8 || W % 32 || W < 32 || col + 3 * W > N || n1 < 0 || n1 > M || n1 > 65535 || n_segs < 0 ||
      n_segs > 65535 || (n1 < M && n_segs < 1) || (n1 < M && slices != 1))
    return -1;
  GruParams p{part, slices, M, N, col, W, bias_a, bias_u, req, pos, segs, n1, mult, state, out, ldo};
  cudaStream_t st = (cudaStream_t)stream;
  int rc = 0;
  if (n1)
    rc = f32 ? b2_launch(mingru_rows_kernel<float>, dim3((W + 127) / 128, n1), dim3(128), 0, st, true, p)
             : b2_launch(mingru_rows_kernel<__nv_bfloat16>, dim3((W + 127) / 128, n1), dim3(128), 0, st, true, p);
  if (rc || n1 == M) return rc;
  // not started while the kernel before still runs: its few, long CTAs would gather on the SMs that happen to be free
  return f32 ? b2_launch(mingru_segments_kernel<float>, dim3(W / 32, n_segs), dim3(kParts * 32), 0, st, false, p)
             : b2_launch(mingru_segments_kernel<__nv_bfloat16>, dim3(W / 32, n_segs), dim3(kParts * 32), 0, st, false, p);
}

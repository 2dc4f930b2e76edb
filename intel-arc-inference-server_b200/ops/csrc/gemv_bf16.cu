// Linears over unquantised weights for a few activation rows, and the 32-bit forms of every linear.
//
//   gemv_bf16_kernel   out = x W^T for up to 16 rows x and a bf16 weight [N][K], weight-streaming.  A CTA owns 32 weight
//                      rows; its four warps take the 64-k steps of the CTA's K range in turn, each with a per-lane
//                      cp.async ring of its own, and meet in shared memory.  The products run on mma.m16n8k16 with the
//                      activations as A and the weight rows as B, in a k order chosen so that a lane's 16-byte vector is
//                      its fragment (as in the lm_head kernel).  The first weight vectors are requested before the
//                      kernel waits for its predecessor.
//                      Epilogues: fp32 slices [split][m][N] (the consumer folds them), bf16, relu(x)^2 as bf16, or SiLU(gate) *
//                      up (or another gated product) over interleave16 rows.  Batched form: batch b multiplies activation row b / x_div with the weight of
//                      expert ids[b] (mixture-of-experts decode rows).
//   linear_f32_kernel  C[M][N] = A[M][K] B[N][K]^T in fp32 FMA arithmetic (models served in 32-bit)
//   linear_f32_rows    the batched expert form of it: one warp per output
//   glu_rows_f32       gated product of interleave16 columns
//
// The role of the reference's bf16 GEMV (src/kernels/gemv_bf16.cl).
#include "common.cuh"

using namespace b2;

namespace {

enum Epi : int { EPI_PART = 0, EPI_BF16 = 1, EPI_SILU = 2, EPI_GLU = 3, EPI_RELU2 = 4 };

struct GemvBfParams {
  const __nv_bfloat16* w;    // [N][K], or [E][N][K] in the batched form
  const int* ids;            // batched form: expert of every batch
  const __nv_bfloat16* x;    // [rows][ldx]
  void* out;
  int M, N, K, ldx, splits, epi, x_div;
  int plane_rows, planes;    // planes > 1: weight rows n read activations of plane min(n / plane_rows, planes - 1),
  long long plane;           // planes this many elements apart
  Glu glu;                   // EPI_GLU
};

constexpr int kStages = 4, kWarps = 4, NG = 4, KU = 2;

template <int MH>
constexpr int stage_bytes() { return (KU * NG + KU * MH) * 512; }
template <int MH>
constexpr int gemv_smem() { return kWarps * kStages * stage_bytes<MH>(); }

// MH: halves of 8 activation rows (1: up to 8 rows, 2: up to 16)
template <int MH>
__global__ void __launch_bounds__(kWarps * 32) gemv_bf16_kernel(const GemvBfParams p) {
  extern __shared__ __align__(16) unsigned char ring_smem[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int n0 = blockIdx.x * 32, split = blockIdx.y, batch = blockIdx.z;
  const bool batched = p.ids != nullptr;
  pdl_launch_dependents();
  if (batched) pdl_wait();     // the expert ids come from the kernel before
  const __nv_bfloat16* w = p.w + (batched ? (size_t)p.ids[batch] * p.N * p.K : 0);
  const int row_x = batched ? batch / p.x_div : 0;
  const int M = batched ? 1 : p.M;
  const int steps_all = p.K / 64;
  const int per = (steps_all + p.splits - 1) / p.splits;
  const int s_lo = split * per, s_hi = min(steps_all, s_lo + per);
  const int steps = max(0, (s_hi - s_lo - warp + kWarps - 1) / kWarps);    // this warp's: s_lo + warp + kWarps * i
  const __nv_bfloat16* wp[NG];
#pragma unroll
  for (int i = 0; i < NG; ++i) wp[i] = w + (size_t)min(n0 + 8 * i + g, p.N - 1) * p.K + t * 8;
  const __nv_bfloat16* x = p.x + (p.planes > 1 ? min(n0 / p.plane_rows, p.planes - 1) * p.plane : 0);
  const __nv_bfloat16* xr[MH];
#pragma unroll
  for (int h = 0; h < MH; ++h) xr[h] = x + (size_t)(row_x + min(8 * h + g, M - 1)) * p.ldx + t * 8;
  constexpr int SB = stage_bytes<MH>();
  unsigned char* ring = ring_smem + warp * kStages * SB + lane * 16;
  const uint32_t ring_s = smem_u32(ring);
  auto issue_w = [&](int i) {
    if (i < steps) {
      const int k = (s_lo + warp + kWarps * i) * 64;
      const uint32_t dst = ring_s + (i % kStages) * SB;
#pragma unroll
      for (int u = 0; u < KU; ++u)
#pragma unroll
        for (int j = 0; j < NG; ++j)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + (u * NG + j) * 512), "l"(wp[j] + k + 32 * u) : "memory");
    }
  };
  auto issue_x = [&](int i) {
    if (i < steps) {
      const int k = (s_lo + warp + kWarps * i) * 64;
      const uint32_t dst = ring_s + (i % kStages) * SB + KU * NG * 512;
#pragma unroll
      for (int u = 0; u < KU; ++u)
#pragma unroll
        for (int h = 0; h < MH; ++h)
          asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"(dst + (u * MH + h) * 512), "l"(xr[h] + k + 32 * u) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");   // an empty group past the end keeps the count uniform
  };
  float acc[NG][4];
#pragma unroll
  for (int i = 0; i < NG; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll
  for (int i = 0; i < kStages; ++i) issue_w(i);
  if (!batched) pdl_wait();
#pragma unroll
  for (int i = 0; i < kStages; ++i) issue_x(i);
  for (int i = 0; i < steps; ++i) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kStages - 1) : "memory");
    const uint4* st = reinterpret_cast<const uint4*>(ring + (i % kStages) * SB);
#pragma unroll
    for (int u = 0; u < KU; ++u) {
      const uint4 av = st[(KU * NG + u * MH) * 32];
      const uint4 bv = MH == 2 ? st[(KU * NG + u * MH + MH - 1) * 32] : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int j = 0; j < NG; ++j) {
        const uint4 wv = st[(u * NG + j) * 32];
        mma_bf16_16816(acc[j], av.x, bv.x, av.y, bv.y, wv.x, wv.y);
        mma_bf16_16816(acc[j], av.z, bv.z, av.w, bv.w, wv.z, wv.w);
      }
    }
    issue_w(i + kStages);   // into the stage just read: its values sit in MMA operands by now
    issue_x(i + kStages);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();          // every warp is done with its ring: the sums reuse it
  float* red = reinterpret_cast<float*>(ring_smem);      // [warp][16 rows][33]
#pragma unroll
  for (int j = 0; j < NG; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) red[(warp * 16 + g + 8 * (e >> 1)) * 33 + 8 * j + 2 * t + (e & 1)] = acc[j][e];
  __syncthreads();
  if (p.epi == EPI_SILU || p.epi == EPI_GLU) {
    for (int i = threadIdx.x; i < M * 16; i += kWarps * 32) {
      const int m = i >> 4, c = i & 15;
      float gt = 0.f, up = 0.f;
#pragma unroll
      for (int q = 0; q < kWarps; ++q) {
        gt += red[(q * 16 + m) * 33 + c];
        up += red[(q * 16 + m) * 33 + 16 + c];
      }
      if (p.epi == EPI_GLU && p.glu.bias) {
        gt += p.glu.bias[n0 + c];
        up += p.glu.bias[n0 + 16 + c];
      }
      if (n0 + 16 + c < p.N)
        reinterpret_cast<__nv_bfloat16*>(p.out)[(size_t)(batched ? batch : m) * (p.N / 2) + n0 / 2 + c] = __float2bfloat16(p.epi == EPI_GLU ? glu(p.glu, gt, up) : silu(gt) * up);
    }
    return;
  }
  for (int i = threadIdx.x; i < M * 32; i += kWarps * 32) {
    const int m = i >> 5, c = i & 31;
    float v = 0.f;
#pragma unroll
    for (int q = 0; q < kWarps; ++q) v += red[(q * 16 + m) * 33 + c];
    if (n0 + c >= p.N) continue;
    if (p.epi == EPI_BF16 || p.epi == EPI_RELU2)
      reinterpret_cast<__nv_bfloat16*>(p.out)[(size_t)(batched ? batch : m) * p.N + n0 + c] = __float2bfloat16(p.epi == EPI_BF16 ? v : relu2(v));
    else if (batched)
      reinterpret_cast<float*>(p.out)[((size_t)batch * p.splits + split) * p.N + n0 + c] = v;
    else
      reinterpret_cast<float*>(p.out)[((size_t)split * M + m) * p.N + n0 + c] = v;
  }
}

// ------------------------------------------------------------------ 32-bit linears
// 64 x 64 tile, 256 threads, 4 x 4 outputs per thread, K in steps of 16
__global__ void __launch_bounds__(256) linear_f32_kernel(const float* __restrict__ a, const float* __restrict__ b,
                                                         float* __restrict__ c, int M, int N, int K, int ldc, int squared) {
  __shared__ float as[16][68], bs[16][68];
  pdl_wait();
  pdl_launch_dependents();
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += 16) {
    float4 av = make_float4(0.f, 0.f, 0.f, 0.f), bv = av;
    if (m0 + lr < M) av = *reinterpret_cast<const float4*>(a + (size_t)(m0 + lr) * K + k0 + lk);
    if (n0 + lr < N) bv = *reinterpret_cast<const float4*>(b + (size_t)(n0 + lr) * K + k0 + lk);
    __syncthreads();
    as[lk][lr] = av.x; as[lk + 1][lr] = av.y; as[lk + 2][lr] = av.z; as[lk + 3][lr] = av.w;
    bs[lk][lr] = bv.x; bs[lk + 1][lr] = bv.y; bs[lk + 2][lr] = bv.z; bs[lk + 3][lr] = bv.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { x[i] = as[k][ty * 4 + i]; y[i] = bs[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (m0 + ty * 4 + i < M && n0 + tx * 4 + j < N) c[(size_t)(m0 + ty * 4 + i) * ldc + n0 + tx * 4 + j] = squared ? relu2(acc[i][j]) : acc[i][j];
}

// batch b: out[b][n] = x[b / x_div] . w[ids[b]][n]; one warp per output.  act 1: SiLU(gate) * up of w rows interleave16, out
// [b][N / 2]; 2: relu(x)^2
__global__ void __launch_bounds__(256) linear_f32_rows_kernel(const float* __restrict__ w, const int* __restrict__ ids,
                                                              const float* __restrict__ x, float* __restrict__ out, int N,
                                                              int K, int ldx, int x_div, int act) {
  const bool do_silu = act == 1;
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, b = blockIdx.y;
  const int outs = do_silu ? N / 2 : N, o = blockIdx.x * 8 + warp;
  if (o >= outs) return;
  const float* we = w + (size_t)ids[b] * N * K;
  const float* xr = x + (size_t)(b / x_div) * ldx;
  const int r0 = do_silu ? (o >> 4) * 32 + (o & 15) : o;
  float u = 0.f, v = 0.f;
  for (int k = lane; k < K; k += 32) {
    u = fmaf(we[(size_t)r0 * K + k], xr[k], u);
    if (do_silu) v = fmaf(we[(size_t)(r0 + 16) * K + k], xr[k], v);
  }
  u = warp_sum(u);
  v = warp_sum(v);
  if (lane == 0) out[(size_t)b * outs + o] = do_silu ? u / (1.f + expf(-u)) * v : act == 2 ? relu2(u) : u;
}

__global__ void __launch_bounds__(256) glu_rows_f32_kernel(const float* __restrict__ in, float* __restrict__ out, int N, const Glu p) {
  pdl_wait();
  pdl_launch_dependents();
  const int o = blockIdx.x * 256 + threadIdx.x;
  if (o >= N / 2) return;
  const float* r = in + (size_t)blockIdx.y * N + (o >> 4) * 32 + (o & 15);
  float g = r[0], u = r[16];
  if (p.bias) {
    g += p.bias[(o >> 4) * 32 + (o & 15)];
    u += p.bias[(o >> 4) * 32 + (o & 15) + 16];
  }
  g = fminf(g, p.limit);
  u = fminf(fmaxf(u, -p.limit), p.limit);
  out[(size_t)blockIdx.y * (N / 2) + o] = g / (1.f + expf(p.gelu ? -gelu_arg(g) : -p.alpha * g)) * (u + p.shift);
}

int sm_count() {
  static int n[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!n[dev & 63]) cudaDeviceGetAttribute(&n[dev & 63], cudaDevAttrMultiProcessorCount, dev);
  return n[dev & 63];
}

template <int MH>
int launch_gemv(const GemvBfParams& p, int batches, cudaStream_t st) {
  static bool configured[64] = {};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(gemv_bf16_kernel<MH>, cudaFuncAttributeMaxDynamicSharedMemorySize, gemv_smem<MH>());
    if (e != cudaSuccess) return (int)e;
    configured[dev & 63] = true;
  }
  return b2_launch(gemv_bf16_kernel<MH>, dim3((p.N + 31) / 32, p.splits, batches), dim3(kWarps * 32), gemv_smem<MH>(), st,
                   true, p);
}

}  // namespace

// K splits over CTAs for a weight [N][K]: enough CTAs for two per SM, at least two 64-k steps per warp.  A function of
// the weight's shape only, so a row's bits do not depend on its company.
extern "C" int b2_gemv_bf16_splits(int N, int K) {
  const int tiles = (N + 31) / 32, steps = K / 64;
  int want = (2 * 148 + tiles - 1) / tiles;
  int most = steps / (2 * kWarps);
  if (most < 1) most = 1;
  if (want > most) want = most;
  if (want > 8) want = 8;
  const int per = (steps + want - 1) / want;
  return (steps + per - 1) / per;       // no empty slices
}

// out: epi 0: fp32 [splits][M][N] (batched: [batch][splits][N]); epi 1, 4: bf16 [M][N]; epi 2: bf16 [M][N / 2] (all splits = 1)
extern "C" int b2_gemv_bf16(const void* w, const int* ids, int batches, const void* x, int ldx, int x_div, void* out, int M,
                            int N, int K, int splits, int epi, void* stream) {
  if (K % 64 || N < 1 || M < 1 || M > 16 || splits < 1 || ldx % 8 || (epi != EPI_PART && splits != 1)) return -1;
  if ((epi == EPI_SILU && N % 32) || epi < EPI_PART || epi > EPI_RELU2 || epi == EPI_GLU) return -2;
  if (ids && (M != 1 || x_div < 1)) return -3;
  GemvBfParams p{(const __nv_bfloat16*)w, ids, (const __nv_bfloat16*)x, out, M, N, K, ldx, splits, epi, x_div, 0, 1, 0, {}};
  return M <= 8 ? launch_gemv<1>(p, ids ? batches : 1, (cudaStream_t)stream)
                : launch_gemv<2>(p, ids ? batches : 1, (cudaStream_t)stream);
}

// epi 0 with activations in `planes` planes (`plane` elements apart) of M rows each: weight rows n read plane
// min(n / plane_rows, planes - 1)
extern "C" int b2_gemv_bf16_planes(const void* w, const void* x, int ldx, int plane_rows, int planes, long long plane, void* out, int M,
                                   int N, int K, int splits, void* stream) {
  if (K % 64 || N < 1 || M < 1 || M > 16 || splits < 1 || ldx % 8 || plane_rows % 32 || plane_rows < 32 || planes < 1 || plane % 8) return -1;
  GemvBfParams p{(const __nv_bfloat16*)w, nullptr, (const __nv_bfloat16*)x, out, M, N, K, ldx, splits, EPI_PART, 1, plane_rows, planes, plane, {}};
  return M <= 8 ? launch_gemv<1>(p, 1, (cudaStream_t)stream) : launch_gemv<2>(p, 1, (cudaStream_t)stream);
}

// bf16 out [M][N / 2] = gated product of the interleave16 columns of x W^T (common.cuh, Glu)
extern "C" int b2_gemv_bf16_glu(const void* w, const void* x, int ldx, void* out, int M, int N, int K, float limit, float alpha,
                                float shift, int gelu, const float* bias, void* stream) {
  if (K % 64 || N % 32 || M < 1 || M > 16 || ldx % 8) return -1;
  GemvBfParams p{(const __nv_bfloat16*)w, nullptr, (const __nv_bfloat16*)x, out, M, N, K, ldx, 1, EPI_GLU, 1, 0, 1, 0,
                 {limit, alpha, shift, gelu, bias}};
  return M <= 8 ? launch_gemv<1>(p, 1, (cudaStream_t)stream) : launch_gemv<2>(p, 1, (cudaStream_t)stream);
}

// in fp32 [M][N] interleave16 -> out [M][N / 2]
extern "C" int b2_glu_rows_f32(const float* in, float* out, int M, int N, float limit, float alpha, float shift, int gelu,
                               const float* bias, void* stream) {
  if (M < 1 || M > 65535 || N % 32) return -1;
  return b2_launch(glu_rows_f32_kernel, dim3((N / 2 + 255) / 256, M), dim3(256), 0, (cudaStream_t)stream, true, in, out, N,
                   Glu{limit, alpha, shift, gelu, bias});
}

extern "C" int b2_linear_f32(const float* a, const float* w, float* c, int M, int N, int K, int ldc, int squared, void* stream) {
  if (K % 16 || M < 1 || N < 1 || ldc < N) return -1;
  return b2_launch(linear_f32_kernel, dim3((N + 63) / 64, (M + 63) / 64), dim3(256), 0, (cudaStream_t)stream, true, a, w, c,
                   M, N, K, ldc, squared);
}

extern "C" int b2_linear_f32_rows(const float* w, const int* ids, int batches, const float* x, int ldx, int x_div, float* out,
                                  int N, int K, int act, void* stream) {
  if (batches < 1 || batches > 65535 || x_div < 1 || act < 0 || act > 2 || (act == 1 && N % 32)) return -1;
  const int outs = act == 1 ? N / 2 : N;
  return b2_launch(linear_f32_rows_kernel, dim3((outs + 7) / 8, batches), dim3(256), 0, (cudaStream_t)stream, true, w, ids, x,
                   out, N, K, ldx, x_div, act);
}

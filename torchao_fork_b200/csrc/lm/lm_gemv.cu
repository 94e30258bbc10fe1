// Products of few rows (decoded tokens) with a bf16 weight matrix: out[t][m] = f(sum_k w[m][k] x[t][k]), fp32 accumulation, read
// at the speed of the weights.  A group of warps owns kRows weight rows and shares out their k; every thread keeps kRows x kFlight
// 16-byte loads in flight and uses each weight for all tokens of the step, whose own values come from L1 (a thread reads the
// same k of every weight row, so nothing is staged).  The groups' partial sums meet in shared memory.  The first round of
// weights is fetched before the kernel waits for the launch in front of it: they depend on nothing.
#include "lm_common.cuh"

using namespace lm;

namespace {

constexpr int kThreads = 256;
constexpr int kRows = 4;

struct GemvArgs {
  const __nv_bfloat16 *x, *w;
  int64_t ld_x, ld_w, ld_out;
  int n, M, K8;                 // K8: 16-byte pieces of a row
  void* out;
};

__device__ __forceinline__ void widen(const uint4& u, float (&f)[8]) { unpack16(u, f, static_cast<const __nv_bfloat16*>(nullptr)); }
// weights pass through once: they do not displace the step's small tensors from L1
__device__ __forceinline__ uint4 ld_stream(const uint4* p) {
  uint4 r;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(r.x), "=r"(r.y), "=r"(r.z), "=r"(r.w) : "l"(p));
  return r;
}

// N: tokens (at least a.n); ACT 0: fp32 result, 1: squared ReLU in bf16
template <int N, int WPG, int ACT>
__global__ void __launch_bounds__(kThreads) gemv_rows_kernel(GemvArgs a) {
  constexpr int kFlight = N <= 2 ? 4 : 2, TG = WPG * 32, GROUPS = kThreads / TG;
  __shared__ float part[GROUPS][WPG][kRows * N];
  const int group = threadIdx.x / TG, tg = threadIdx.x % TG, lane = threadIdx.x & 31, wg = tg / 32;
  const int m0 = (blockIdx.x * GROUPS + group) * kRows;
  const uint4* wr[kRows];
#pragma unroll
  for (int r = 0; r < kRows; ++r) wr[r] = reinterpret_cast<const uint4*>(a.w + (int64_t)min(m0 + r, a.M - 1) * a.ld_w);
  float acc[kRows][N];
#pragma unroll
  for (int r = 0; r < kRows; ++r)
#pragma unroll
    for (int t = 0; t < N; ++t) acc[r][t] = 0.f;
  pdl_trigger();
  uint4 v[kFlight][kRows];
  auto fetch = [&](int k) {
#pragma unroll
    for (int u = 0; u < kFlight; ++u)
#pragma unroll
      for (int r = 0; r < kRows; ++r) v[u][r] = k + u * TG < a.K8 ? ld_stream(wr[r] + k + u * TG) : make_uint4(0, 0, 0, 0);
  };
  fetch(tg);
  pdl_wait();
  for (int k = tg; k < a.K8; k += TG * kFlight) {
    if (k != tg) fetch(k);
#pragma unroll
    for (int u = 0; u < kFlight; ++u) {
      if (k + u * TG >= a.K8) break;
      float wf[kRows][8];
#pragma unroll
      for (int r = 0; r < kRows; ++r) widen(v[u][r], wf[r]);
#pragma unroll
      for (int t = 0; t < N; ++t) {
        float xf[8];
        widen(*(reinterpret_cast<const uint4*>(a.x + (int64_t)min(t, a.n - 1) * a.ld_x) + k + u * TG), xf);
#pragma unroll
        for (int r = 0; r < kRows; ++r)
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[r][t] = fmaf(wf[r][e], xf[e], acc[r][t]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < kRows; ++r)
#pragma unroll
    for (int t = 0; t < N; ++t) {
      const float s = warp_sum(acc[r][t]);
      if (lane == 0) part[group][wg][t * kRows + r] = s;
    }
  __syncthreads();
  for (int i = tg; i < kRows * N; i += TG) {
    const int t = i / kRows, m = m0 + i % kRows;
    if (t >= a.n || m >= a.M) continue;
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < WPG; ++w) s += part[group][w][i];
    if (ACT == 1) {
      s = fmaxf(s, 0.f);
      static_cast<__nv_bfloat16*>(a.out)[t * a.ld_out + m] = __float2bfloat16_rn(s * s);
    } else {
      static_cast<float*>(a.out)[t * a.ld_out + m] = s;
    }
  }
}

template <int N, int ACT>
int launch(const GemvArgs& a, cudaStream_t st) {
  // warps that share out a weight row: enough for two or so pieces in flight each, more when there are few rows
  int wpg = 1;
  while (wpg < 8 && (a.K8 > 32 * wpg * 8 || (a.K8 > 32 * wpg * 2 && (int64_t)(a.M + kRows - 1) / kRows * wpg < 148 * 16))) wpg *= 2;
  const unsigned groups = (unsigned)((a.M + kRows - 1) / kRows), per = 8 / wpg;
  const dim3 grid((groups + per - 1) / per), block(kThreads);
  if (wpg == 1) return lm_launch_early(gemv_rows_kernel<N, 1, ACT>, grid, block, 0, st, a);
  if (wpg == 2) return lm_launch_early(gemv_rows_kernel<N, 2, ACT>, grid, block, 0, st, a);
  if (wpg == 4) return lm_launch_early(gemv_rows_kernel<N, 4, ACT>, grid, block, 0, st, a);
  return lm_launch_early(gemv_rows_kernel<N, 8, ACT>, grid, block, 0, st, a);
}

template <int ACT>
int launch_n(const GemvArgs& a, cudaStream_t st) {
  if (a.n == 1) return launch<1, ACT>(a, st);
  if (a.n == 2) return launch<2, ACT>(a, st);
  if (a.n <= 4) return launch<4, ACT>(a, st);
  return launch<8, ACT>(a, st);
}

}  // namespace

extern "C" int ao_lm_gemv_rows(const void* x, int64_t ld_x, const void* w, int64_t ld_w, int64_t n, int64_t M, int64_t K, int act, void* out,
                               int64_t ld_out, void* stream) {
  LM_CHECK_ARG(x && w && out && n > 0 && M > 0 && K > 0 && ld_x >= K && ld_w >= K && ld_out >= M && (act == 0 || act == 1));
  LM_CHECK_ARG(M <= (1 << 30) && K <= (1 << 30));
  if (n > 8 || K % 8 || ld_x % 8 || ld_w % 8 || reinterpret_cast<uintptr_t>(x) % 16 || reinterpret_cast<uintptr_t>(w) % 16)
    return AO_B200_ERR_UNSUPPORTED;
  const GemvArgs a{static_cast<const __nv_bfloat16*>(x), static_cast<const __nv_bfloat16*>(w), ld_x, ld_w, ld_out, (int)n, (int)M, (int)(K / 8), out};
  return act ? launch_n<1>(a, lm_stream(stream)) : launch_n<0>(a, lm_stream(stream));
}

// Gated delta rule: a matrix state per head that forgets by one factor per token and, before a token is written, takes out
// what the state already answers to its key,
//     S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q.
// Every value column of S is a recurrence of its own (u and o of a column need that column only), so a group of lanes owns a
// column: LPC lanes hold its d entries in registers, the two products S^T k and S^T q are sums over the group.
//
// Tokens are folded in B at a time.  With G_j the product of the decays of the block's tokens 0 .. j and R_ij that of tokens
// i + 1 .. j (products only, nothing is divided by a decay), all of a block's 2 B products meet the state S it starts from,
//     u_j = beta_j (v_j - G_j S^T k_j - sum_{i<j} R_ij (k_i . k_j) u_i),
//     o_j = G_j S^T q_j + sum_{i<=j} R_ij (k_i . q_j) u_i,
//     S'  = G_last S + sum_i R_i,last k_i u_i^T,
// which is the token-by-token recurrence with the sums in another order: the reductions over a group of lanes, the long part
// of a token's latency, run for B tokens at once.  The B^2 scalars of a block are the same for all columns of a head and are
// made once per CTA.  Everything is fp32.
//
// In front of it: the causal convolutions over time with SiLU, unit queries and keys, decays and step sizes, per row.
#include "lm_common.cuh"

using namespace lm;

namespace {

constexpr int kWarps = 4;

__device__ __forceinline__ void cp_async4(void* smem, const void* gmem) {
  const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(s), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
}

struct DeltaArgs {
  const float* qk;               // [n][2][G][dp]: unit queries (scaled), unit keys; zeros beyond d
  const float* v;                // [n][H dv]
  const float* gb;               // [n][H][2]: decay, step size
  int H, G, dp, dv;
  float* state;                  // [slots][H][dv][dp]: a value column's entries are neighbours
  const int32_t *slot, *pos, *seg_first, *seg_count;
  const float* conv_x;           // the convolutions' inputs [n][ld_conv], `channels` of them: the last taps - 1 become the slot's memory
  int64_t ld_conv, channels;
  int taps;
  float* conv_state;             // [slots][taps - 1][channels]
  float* out;                    // [n][H dv]
};

// scalars of a block of B tokens, in shared memory: [kk: B x B][kq: B x B][G_j][R_j,last][beta_j]
template <int B>
struct Scalars {
  static constexpr int kKK = 0, kKQ = B * B, kG = 2 * B * B, kE = kG + B, kBeta = kE + B, kSize = kBeta + B;
};

template <int DR4, int LPC, int B, int TS>   // float4 pieces per lane, lanes per column, tokens per block, tokens staged at a time
__global__ void __launch_bounds__(kWarps * 32) delta_recurrence_kernel(DeltaArgs A) {
  constexpr int CW = 32 / LPC, CC = kWarps * CW;      // value columns per warp / per CTA
  constexpr int D = LPC * DR4 * 4;                    // key size covered
  constexpr int SC = (Scalars<B>::kSize + 3) / 4 * 4, NB = TS / B;
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;                                     // [2][TS][D]
  float* ks = qs + 2 * TS * D;                        // [2][TS][D]
  float* vs = ks + 2 * TS * D;                        // [2][TS][CC]
  float* gb = vs + 2 * TS * CC;                       // [2][TS][2]
  float* scal = gb + 2 * TS * 2;                      // [NB][SC]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, p = lane % LPC, grp = lane / LPC;
  const int seg = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * CC;
  const int first = A.seg_first[seg], count = A.seg_count[seg];
  const int g = h / (A.H / A.G), dp = A.dp, dv = A.dv;
  const int cl = warp * CW + grp, c = c0 + cl;        // this lane group's column: in the CTA, in the head
  const bool fresh = A.pos[first] == 0;
  float* srow = A.state + (((int64_t)A.slot[first] * A.H + h) * dv + c) * dp;
  float4 S[DR4];
#pragma unroll
  for (int r = 0; r < DR4; ++r) {
    const int i = 4 * (p + LPC * r);
    S[r] = (!fresh && c < dv && i < dp) ? *reinterpret_cast<const float4*>(srow + i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (dp < D)   // the key entries beyond dp are never staged: zeros in both buffers
    for (int i = tid; i < 2 * TS * (D - dp); i += kWarps * 32) {
      const int j = i / (D - dp), e = dp + i - j * (D - dp);
      qs[j * D + e] = ks[j * D + e] = 0.f;
    }
  const int pieces = dp / 4;
  auto stage = [&](int t0, int buf) {                 // tokens t0 .. + TS; past the segment: decay 1, step 0, zero vectors
    for (int i = tid; i < TS * pieces; i += kWarps * 32) {
      const int j = i / pieces, e = (i - j * pieces) * 4;
      float* dq = qs + (buf * TS + j) * D + e;
      float* dk = ks + (buf * TS + j) * D + e;
      if (t0 + j < count) {
        const float* src = A.qk + (((int64_t)(first + t0 + j) * 2) * A.G + g) * dp + e;
        cp_async16(dq, src);
        cp_async16(dk, src + (int64_t)A.G * dp);
      } else {
        *reinterpret_cast<float4*>(dq) = *reinterpret_cast<float4*>(dk) = make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
    for (int i = tid; i < TS * CC; i += kWarps * 32) {
      const int j = i / CC, e = i - j * CC;
      float* d = vs + buf * TS * CC + i;
      if (t0 + j < count && c0 + e < dv)
        cp_async4(d, A.v + (int64_t)(first + t0 + j) * A.H * dv + (int64_t)h * dv + c0 + e);
      else
        *d = 0.f;
    }
    for (int i = tid; i < TS * 2; i += kWarps * 32) {
      float* d = gb + buf * TS * 2 + i;
      if (t0 + i / 2 < count)
        cp_async4(d, A.gb + ((int64_t)(first + t0 + i / 2) * A.H + h) * 2 + (i & 1));
      else
        *d = (i & 1) ? 0.f : 1.f;
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  stage(0, 0);
  int buf = 0;
  for (int t0 = 0; t0 < count; t0 += TS, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();            // this stage is in place; nobody reads the other buffer or the old scalars any more
    if (t0 + TS < count) stage(t0 + TS, buf ^ 1);
    const float* kb = ks + buf * TS * D;
    const float* qb = qs + buf * TS * D;
    const float* gbb = gb + buf * TS * 2;
    // the blocks' scalars: a group of lanes per pair (i, j) of a block, i <= j
    constexpr int kPairs = B * (B + 1) / 2;
    for (int w0 = warp * CW; w0 < NB * kPairs; w0 += kWarps * CW) {      // uniform over the warp
      const int wi = min(w0 + grp, NB * kPairs - 1), blk = wi / kPairs;
      int rem = wi - blk * kPairs, j = 0;
      while (rem > j) rem -= ++j;                                         // pair number -> (i = rem, j)
      const int i = rem;
      const float* ki = kb + (blk * B + i) * D;
      const float* kj = kb + (blk * B + j) * D;
      const float* qj = qb + (blk * B + j) * D;
      float kk = 0.f, kq = 0.f;
#pragma unroll
      for (int r = 0; r < DR4; ++r) {
        const int e = 4 * (p + LPC * r);
        const float4 x = *reinterpret_cast<const float4*>(ki + e), y = *reinterpret_cast<const float4*>(kj + e),
                     z = *reinterpret_cast<const float4*>(qj + e);
        kk = fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, kk))));
        kq = fmaf(x.x, z.x, fmaf(x.y, z.y, fmaf(x.z, z.z, fmaf(x.w, z.w, kq))));
      }
#pragma unroll
      for (int o = LPC / 2; o > 0; o >>= 1) {
        kk += __shfl_xor_sync(0xffffffffu, kk, o);
        kq += __shfl_xor_sync(0xffffffffu, kq, o);
      }
      if (p == 0 && w0 + grp < NB * kPairs) {
        float dec = 1.f;
        for (int m = i + 1; m <= j; ++m) dec *= gbb[2 * (blk * B + m)];
        float* sc = scal + blk * SC;
        sc[Scalars<B>::kKK + i * B + j] = dec * kk;
        sc[Scalars<B>::kKQ + i * B + j] = dec * kq;
      }
    }
    for (int w = tid; w < TS; w += kWarps * 32) {
      const int blk = w / B, j = w - blk * B;
      float pre = 1.f, post = 1.f;
      for (int m = 0; m <= j; ++m) pre *= gbb[2 * (blk * B + m)];
      for (int m = j + 1; m < B; ++m) post *= gbb[2 * (blk * B + m)];
      float* sc = scal + blk * SC;
      sc[Scalars<B>::kG + j] = pre;
      sc[Scalars<B>::kE + j] = post;
      sc[Scalars<B>::kBeta + j] = gbb[2 * w + 1];
    }
    __syncthreads();
    const int nblk = (min(TS, count - t0) + B - 1) / B;
    for (int blk = 0; blk < nblk; ++blk) {
      const float* sc = scal + blk * SC;
      float4 k[B][DR4];
      float a[B], b[B];
#pragma unroll
      for (int j = 0; j < B; ++j) {
        float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
#pragma unroll
        for (int r = 0; r < DR4; ++r) {
          const int e = 4 * (p + LPC * r);
          k[j][r] = *reinterpret_cast<const float4*>(kb + (blk * B + j) * D + e);
          const float4 q = *reinterpret_cast<const float4*>(qb + (blk * B + j) * D + e);
          a0 = fmaf(S[r].x, k[j][r].x, a0), a1 = fmaf(S[r].y, k[j][r].y, a1);
          a0 = fmaf(S[r].z, k[j][r].z, a0), a1 = fmaf(S[r].w, k[j][r].w, a1);
          b0 = fmaf(S[r].x, q.x, b0), b1 = fmaf(S[r].y, q.y, b1);
          b0 = fmaf(S[r].z, q.z, b0), b1 = fmaf(S[r].w, q.w, b1);
        }
        a[j] = a0 + a1, b[j] = b0 + b1;
      }
#pragma unroll
      for (int o = LPC / 2; o > 0; o >>= 1) {
#pragma unroll
        for (int j = 0; j < B; ++j) {
          a[j] += __shfl_xor_sync(0xffffffffu, a[j], o);
          b[j] += __shfl_xor_sync(0xffffffffu, b[j], o);
        }
      }
      float u[B];
#pragma unroll
      for (int j = 0; j < B; ++j) {
        float t = fmaf(-sc[Scalars<B>::kG + j], a[j], vs[(buf * TS + blk * B + j) * CC + cl]);
#pragma unroll
        for (int i = 0; i < j; ++i) t = fmaf(-sc[Scalars<B>::kKK + i * B + j], u[i], t);
        u[j] = sc[Scalars<B>::kBeta + j] * t;
      }
      float mine = 0.f;                               // lane j of the group keeps token j's read-out
#pragma unroll
      for (int j = 0; j < B; ++j) {
        float o = sc[Scalars<B>::kG + j] * b[j];
#pragma unroll
        for (int i = 0; i <= j; ++i) o = fmaf(sc[Scalars<B>::kKQ + i * B + j], u[i], o);
        if (p == j) mine = o;
      }
      const float G = sc[Scalars<B>::kG + B - 1];
#pragma unroll
      for (int r = 0; r < DR4; ++r) S[r].x *= G, S[r].y *= G, S[r].z *= G, S[r].w *= G;
#pragma unroll
      for (int j = 0; j < B; ++j) {
        const float w = sc[Scalars<B>::kE + j] * u[j];
#pragma unroll
        for (int r = 0; r < DR4; ++r) {
          S[r].x = fmaf(w, k[j][r].x, S[r].x), S[r].y = fmaf(w, k[j][r].y, S[r].y);
          S[r].z = fmaf(w, k[j][r].z, S[r].z), S[r].w = fmaf(w, k[j][r].w, S[r].w);
        }
      }
      const int t = t0 + blk * B + p;
      if (p < B && t < count && c < dv) A.out[(int64_t)(first + t) * A.H * dv + (int64_t)h * dv + c] = mine;
    }
  }
#pragma unroll
  for (int r = 0; r < DR4; ++r) {
    const int i = 4 * (p + LPC * r);
    if (c < dv && i < dp) *reinterpret_cast<float4*>(srow + i) = S[r];
  }
  if (A.conv_x && A.taps > 1) {   // the segment's CTAs share out the channels of the convolution memory
    const int keep = A.taps - 1;
    const int64_t last = first + count - 1;
    const int p0 = A.pos[first];
    float* st = A.conv_state + (int64_t)A.slot[first] * keep * A.channels;
    const int64_t nth = (int64_t)gridDim.y * gridDim.z * blockDim.x;
    for (int64_t ch = ((int64_t)h * gridDim.z + blockIdx.z) * blockDim.x + tid; ch < A.channels; ch += nth)
      for (int j = 0; j < keep; ++j) {      // ascending: a row of the old memory is read before it is overwritten
        const int s = count - keep + j;     // index among the segment's rows
        float x = 0.f;
        if (s >= 0)
          x = A.conv_x[(last - (keep - 1 - j)) * A.ld_conv + ch];
        else if (p0 + s >= 0)
          x = st[(int64_t)(keep + s) * A.channels + ch];
        st[(int64_t)j * A.channels + ch] = x;
      }
  }
}

template <int DR4, int LPC, int B, int TS>
int launch_delta(const DeltaArgs& A, int n_segments, cudaStream_t st) {
  constexpr int CC = kWarps * (32 / LPC), D = LPC * DR4 * 4, SC = (Scalars<B>::kSize + 3) / 4 * 4;
  constexpr size_t smem = ((size_t)4 * TS * D + 2 * TS * CC + 2 * TS * 2 + (TS / B) * SC) * sizeof(float);
  static_assert(smem <= 200 * 1024 && B <= LPC && TS % B == 0, "");
  auto kern = delta_recurrence_kernel<DR4, LPC, B, TS>;
  if (smem > 48 * 1024) {
    static bool set = false;   // per instantiation
    if (!set) {
      if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return AO_B200_ERR_CUDA;
      set = true;
    }
  }
  kern<<<dim3((unsigned)n_segments, (unsigned)A.H, (unsigned)((A.dv + CC - 1) / CC)), kWarps * 32, smem, st>>>(A);
  return lm_launch_status();
}

// ---------------------------------------------------------------------------------------------------------------
// One warp per (row, unit): a unit is a query head, a key head, 128 value channels, or 32 heads' decays and step sizes.
template <typename T>
__global__ void __launch_bounds__(256) delta_prep_kernel(const float* __restrict__ proj, int64_t ld, int64_t conv_off, int64_t a_off,
                                                         int64_t b_off, int H, int G, int d, int dp, int dv, int taps,
                                                         const T* __restrict__ conv_w, const float* __restrict__ conv_state,
                                                         const int32_t* __restrict__ slot, const int32_t* __restrict__ pos,
                                                         const int32_t* __restrict__ back, const T* __restrict__ a_log,
                                                         const T* __restrict__ dt_bias, float unit_eps, float q_scale,
                                                         float* __restrict__ qk, float* __restrict__ v, float* __restrict__ gb) {
  constexpr int kVals = 8;       // a head of up to 256 entries stays in registers between its sum of squares and its output
  const int64_t t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int bk = back[t], ps = pos[t];
  const int64_t C = (int64_t)2 * G * d + (int64_t)H * dv;
  const float* st = conv_state + (int64_t)slot[t] * (taps > 1 ? taps - 1 : 1) * C;
  const float* x = proj + t * ld + conv_off;
  auto conv = [&](int64_t c) {
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {
      const int delta = taps - 1 - j;     // rows back in time
      float u = 0.f;
      if (delta <= bk)
        u = x[c - (int64_t)delta * ld];
      else if (delta <= ps)
        u = st[(int64_t)(taps - 1 - (delta - bk)) * C + c];
      acc = fmaf(ldf(conv_w + (int64_t)j * C + c), u, acc);
    }
    return acc / (1.f + expf(-acc));
  };
  const int vunits = (H * dv + 127) / 128, gunits = (H + 31) / 32, units = 2 * G + vunits + gunits;
  for (int un = blockIdx.y * 8 + warp; un < units; un += gridDim.y * 8) {
    if (un < 2 * G) {
      const int64_t c0 = (int64_t)un * d;               // [queries | keys] are the first 2 G d channels
      float* dst = qk + (t * 2 * G + un) * dp;
      float val[kVals], ss = 0.f;
#pragma unroll
      for (int e = 0; e < kVals; ++e) {
        const int i = lane + 32 * e;
        val[e] = i < d ? conv(c0 + i) : 0.f;
        ss = fmaf(val[e], val[e], ss);
      }
      for (int i = lane + 32 * kVals; i < d; i += 32) {
        const float y = conv(c0 + i);
        ss = fmaf(y, y, ss);
      }
      const float k = (un < G ? q_scale : 1.f) / sqrtf(warp_sum(ss) + unit_eps);
#pragma unroll
      for (int e = 0; e < kVals; ++e) {
        const int i = lane + 32 * e;
        if (i < dp) dst[i] = val[e] * k;
      }
      for (int i = lane + 32 * kVals; i < dp; i += 32) dst[i] = i < d ? conv(c0 + i) * k : 0.f;
    } else if (un < 2 * G + vunits) {
      const int64_t base = (int64_t)(un - 2 * G) * 128;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int64_t i = base + lane + 32 * e;
        if (i < (int64_t)H * dv) v[t * H * dv + i] = conv((int64_t)2 * G * d + i);
      }
    } else {
      const int h = (un - 2 * G - vunits) * 32 + lane;
      if (h < H) {
        const float z = proj[t * ld + a_off + h] + ldf(dt_bias + h);
        const float soft = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
        gb[(t * H + h) * 2] = expf(-expf(ldf(a_log + h)) * soft);
        gb[(t * H + h) * 2 + 1] = 1.f / (1.f + expf(-proj[t * ld + b_off + h]));
      }
    }
  }
}

}  // namespace

extern "C" int ao_lm_delta_prep(const float* proj, int64_t ld, int64_t conv_off, int64_t a_off, int64_t b_off, int64_t n, int H, int G,
                                int d, int dp, int dv, int taps, const void* conv_w, const float* conv_state, const int32_t* slot,
                                const int32_t* pos, const int32_t* back, const void* a_log, const void* dt_bias, int dt, float unit_eps,
                                float q_scale, float* qk, float* v, float* gb, void* stream) {
  LM_CHECK_ARG(proj && conv_w && conv_state && slot && pos && back && a_log && dt_bias && qk && v && gb);
  LM_CHECK_ARG(n > 0 && H > 0 && G > 0 && H % G == 0 && d > 0 && dp >= d && dp % 4 == 0 && dp < d + 4 && dv > 0 && taps >= 1);
  const int units = 2 * G + (H * dv + 127) / 128 + (H + 31) / 32;
  const unsigned parts = (unsigned)((units + 7) / 8 > 64 ? 64 : (units + 7) / 8);
  LM_DISPATCH(dt, delta_prep_kernel<T><<<dim3((unsigned)n, parts), 256, 0, lm_stream(stream)>>>(
                      proj, ld, conv_off, a_off, b_off, H, G, d, dp, dv, taps, static_cast<const T*>(conv_w), conv_state, slot, pos,
                      back, static_cast<const T*>(a_log), static_cast<const T*>(dt_bias), unit_eps, q_scale, qk, v, gb));
  return lm_launch_status();
}

extern "C" int ao_lm_delta_recurrence(const float* qk, const float* v, const float* gb, int H, int G, int dp, int dv, float* state,
                                      const int32_t* slot, const int32_t* pos, const int32_t* seg_first, const int32_t* seg_count,
                                      int n_segments, int block, const float* conv_x, int64_t ld_conv, int64_t channels, int taps,
                                      float* conv_state, float* out, void* stream) {
  LM_CHECK_ARG(qk && v && gb && state && slot && pos && seg_first && seg_count && out && (!conv_x || conv_state));
  LM_CHECK_ARG(n_segments > 0 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && dp > 0 && dp % 4 == 0 && dv > 0 && taps >= 1);
  LM_CHECK_ARG(reinterpret_cast<uintptr_t>(qk) % 16 == 0 && reinterpret_cast<uintptr_t>(state) % 16 == 0 && (block == 1 || block == 4));
  const DeltaArgs A{qk, v, gb, H, G, dp, dv, state, slot, pos, seg_first, seg_count, conv_x, ld_conv, channels, taps, conv_state, out};
  const cudaStream_t st = lm_stream(stream);
#define LM_DELTA(DR4, LPC, TS) return block == 1 ? launch_delta<DR4, LPC, 1, 4>(A, n_segments, st) : launch_delta<DR4, LPC, 4, TS>(A, n_segments, st)
  if (dp <= 16) LM_DELTA(1, 4, 16);
  if (dp <= 32) LM_DELTA(1, 8, 16);
  if (dp <= 64) LM_DELTA(2, 8, 16);
  if (dp <= 128) LM_DELTA(4, 8, 16);
  if (dp <= 256) LM_DELTA(4, 16, 16);
  if (dp <= 512) LM_DELTA(4, 32, 8);
  if (dp <= 1024) LM_DELTA(8, 32, 8);
#undef LM_DELTA
  return AO_B200_ERR_UNSUPPORTED;
}

// Gated delta rule: a matrix state per head that forgets by one factor per token and, before a token is written, takes out
// what the state already answers to its key,
//     S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q.
// Every value column of S is a recurrence of its own (u and o of a column need that column only), so a group of lanes owns a
// column: LPC lanes hold its d entries in registers, the two products S^T k and S^T q are sums over the group.
//
// Tokens are folded in B at a time (eight; four where a key has more than 256 entries; one for steps of single rows).  With G_j the product of the decays of the block's tokens 0 .. j and R_ij that of tokens
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

__device__ __forceinline__ float dot4(const float4& x, const float4& y, float acc) {
  return fmaf(x.x, y.x, fmaf(x.y, y.y, fmaf(x.z, y.z, fmaf(x.w, y.w, acc))));
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

// Tokens t0 .. t0 + TS of a segment into shared memory by nth threads (asynchronous copies, one group): query and key rows of stride D, the
// CTA's CC value columns from c0 on, decays and step sizes.  Past the segment: decay 1, step 0, zero vectors.
template <int TS, int CC>
__device__ __forceinline__ void stage_tokens(const DeltaArgs& A, int first, int count, int t0, int g, int h, int c0, float* qs,
                                             float* ks, int D, float* vs, float* gb, int tid, int nth) {
  const int pieces = A.dp / 4;
  for (int i = tid; i < TS * pieces; i += nth) {
    const int j = i / pieces, e = (i - j * pieces) * 4;
    if (t0 + j < count) {
      const float* src = A.qk + (((int64_t)(first + t0 + j) * 2) * A.G + g) * A.dp + e;
      cp_async16(qs + j * D + e, src);
      cp_async16(ks + j * D + e, src + (int64_t)A.G * A.dp);
    } else {
      *reinterpret_cast<float4*>(qs + j * D + e) = *reinterpret_cast<float4*>(ks + j * D + e) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  for (int i = tid; i < TS * CC; i += nth) {
    const int j = i / CC, e = i - j * CC;
    if (t0 + j < count && c0 + e < A.dv)
      cp_async4(vs + i, A.v + (int64_t)(first + t0 + j) * A.H * A.dv + (int64_t)h * A.dv + c0 + e);
    else
      vs[i] = 0.f;
  }
  for (int i = tid; i < TS * 2; i += nth) {
    if (t0 + i / 2 < count)
      cp_async4(gb + i, A.gb + ((int64_t)(first + t0 + i / 2) * A.H + h) * 2 + (i & 1));
    else
      gb[i] = (i & 1) ? 0.f : 1.f;
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
}

// The last taps - 1 inputs of the segment's convolutions become the slot's memory; the segment's CTAs share out the channels.
__device__ __forceinline__ void save_conv_memory(const DeltaArgs& A, int first, int count) {
  if (!A.conv_x || A.taps <= 1) return;
  const int keep = A.taps - 1;
  const int64_t last = first + count - 1;
  const int p0 = A.pos[first];
  float* st = A.conv_state + (int64_t)A.slot[first] * keep * A.channels;
  const int64_t nth = (int64_t)gridDim.y * gridDim.z * blockDim.x;
  for (int64_t ch = ((int64_t)blockIdx.y * gridDim.z + blockIdx.z) * blockDim.x + threadIdx.x; ch < A.channels; ch += nth)
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
  auto stage = [&](int t0, int buf) {
    stage_tokens<TS, CC>(A, first, count, t0, g, h, c0, qs + buf * TS * D, ks + buf * TS * D, D, vs + buf * TS * CC, gb + buf * TS * 2, tid, kWarps * 32);
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
  save_conv_memory(A, first, count);
}

// Blocks of eight tokens for key sizes up to 256.  Eight warps per CTA: four fold blocks into the state, two make the blocks'
// scalars one stage ahead, two fetch the rows two stages ahead; one barrier per stage of 16 tokens.
// A group of LPC lanes owns NC = LPC / 8 value columns, so that one load of a key or query piece serves NC products.  A
// lane's slots are permuted by its own number, slot j holding token j ^ t and slot s column s ^ c with (c, t) = lane in the
// group: the sums over the lanes then run as a halving exchange (each step sends the slots that the partner keeps, nothing is
// selected), after which lane (c, t) holds both products of token t with column c.  The triangular system of a block is the
// same for all columns and is inverted once,
//     u = T w,  w_j = beta_j (v_j - G_j S^T k_j),  T = (1 + L)^-1,  L_ji = beta_j R_ij (k_i . k_j) for i < j.
constexpr int kB8 = 8, kRec = 20;      // record of a token t: {beta G, beta, G, E}, {G_last, T[t][t^1] .. T[t][t^7]}, {C[t][t^0] .. C[t][t^7]}

// one warp: the scalars of the block of eight tokens whose keys / queries start at kb / qb (rows of D) -> rec[8][kRec]
template <int D>
__device__ __forceinline__ void block_scalars(const float* kb, const float* qb, const float* gbb, float* rec, float* scratch) {
  constexpr int P = (D + 127) / 128;
  const int lane = threadIdx.x & 31;
  float x[64];                         // k_i . q_j for i <= j (36), then k_i . k_j for i < j (28)
  float4 k[kB8][P];
#pragma unroll
  for (int j = 0; j < kB8; ++j)
#pragma unroll
    for (int r = 0; r < P; ++r) {
      const int e = 4 * (lane + 32 * r);
      k[j][r] = e < D ? *reinterpret_cast<const float4*>(kb + j * D + e) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
  for (int j = 0; j < kB8; ++j) {
    float4 q[P];
#pragma unroll
    for (int r = 0; r < P; ++r) {
      const int e = 4 * (lane + 32 * r);
      q[r] = e < D ? *reinterpret_cast<const float4*>(qb + j * D + e) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i <= j; ++i) {
      float a = 0.f, b = 0.f;
#pragma unroll
      for (int r = 0; r < P; ++r) a = dot4(k[i][r], q[r], a), b = dot4(k[i][r], k[j][r], b);
      x[j * (j + 1) / 2 + i] = a;
      if (i < j) x[36 + j * (j - 1) / 2 + i] = b;
    }
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {   // halve the products with every step: lane l ends with products 2 l and 2 l + 1
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < 2 * o; ++i) {
      const float send = up ? x[i] : x[i + 2 * o], keep = up ? x[i + 2 * o] : x[i];
      x[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
    }
  }
  __syncwarp();
  scratch[2 * lane] = x[0], scratch[2 * lane + 1] = x[1];
  __syncwarp();
  const int t = lane & 7;              // lanes in fours do the same: nothing below waits on a branch
  float gm[kB8], kq[kB8], kk[kB8];
#pragma unroll
  for (int i = 0; i < kB8; ++i) {      // (beyond i = t the loads are valid and unused)
    gm[i] = gbb[2 * i];
    kq[i] = scratch[t * (t + 1) / 2 + min(i, t)];
    kk[i] = scratch[36 + (i < t ? t * (t - 1) / 2 + i : 0)];
  }
  const float be = gbb[2 * t + 1];
  float G = 1.f, all = 1.f, E = 1.f, R = 1.f, C[kB8], Lrow[kB8];
#pragma unroll
  for (int m = 0; m < kB8; ++m) {
    all *= gm[m];
    G *= m <= t ? gm[m] : 1.f;
    E *= m <= t ? 1.f : gm[m];
  }
#pragma unroll
  for (int i = kB8 - 1; i >= 0; --i) { // R = product of the decays of tokens i + 1 .. t
    C[i] = i <= t ? R * kq[i] : 0.f;
    Lrow[i] = i < t ? be * R * kk[i] : 0.f;
    R *= i <= t ? gm[i] : 1.f;
  }
  float* Lm = scratch + 64;            // [8][8]
  float* d = rec + t * kRec;
  if (lane < kB8) {
    *reinterpret_cast<float4*>(Lm + t * 8) = make_float4(Lrow[0], Lrow[1], Lrow[2], Lrow[3]);
    *reinterpret_cast<float4*>(Lm + t * 8 + 4) = make_float4(Lrow[4], Lrow[5], Lrow[6], Lrow[7]);
    *reinterpret_cast<float4*>(d) = make_float4(be * G, be, G, E);
    d[4] = all;
#pragma unroll
    for (int i = 0; i < kB8; ++i) d[12 + (t ^ i)] = C[i];
  }
  __syncwarp();
  float T[kB8], Lr[kB8][kB8];          // column t of T by forward substitution
#pragma unroll
  for (int r = 1; r < kB8; ++r)
#pragma unroll
    for (int m = 0; m < r; m += 4) {
      const float4 l = *reinterpret_cast<const float4*>(Lm + r * 8 + m);
      Lr[r][m] = l.x, Lr[r][m + 1] = l.y, Lr[r][m + 2] = l.z, Lr[r][m + 3] = l.w;
    }
#pragma unroll
  for (int r = 0; r < kB8; ++r) {
    float s = r == t ? 1.f : 0.f;
#pragma unroll
    for (int m = 0; m < r; ++m) s = fmaf(-Lr[r][m], T[m], s);
    T[r] = s;
  }
  if (lane < kB8) {
#pragma unroll
    for (int r = 0; r < kB8; ++r)
      if (r != t) rec[r * kRec + 4 + (r ^ t)] = T[r];
  }
}

template <int DR4, int LPC>
__global__ void __launch_bounds__(256, DR4 == 1 ? 2 : 1) delta_block8_kernel(DeltaArgs A) {
  constexpr int TS = 16, NB = TS / kB8, NC = LPC / 8;
  constexpr int CW = NC * (32 / LPC), CC = kWarps * CW;     // value columns per folding warp / per CTA
  constexpr int D = LPC * DR4 * 4;
  extern __shared__ __align__(16) float sm[];
  float* qs = sm;                                     // [3][TS][D]
  float* ks = qs + 3 * TS * D;                        // [3][TS][D]
  float* vs = ks + 3 * TS * D;                        // [3][TS][CC]
  float* gb = vs + 3 * TS * CC;                       // [3][TS][2]
  float* rec = gb + 3 * TS * 2;                       // [2][TS][kRec]
  float* us = rec + 2 * TS * kRec;                    // [kWarps][CW][8]: decayed u of a block's tokens
  float* scratch = us + kWarps * CW * 8;              // [NB][128]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, p = lane % LPC, grp = lane / LPC;
  const int tb = lane & 7, cb = (lane >> 3) & (NC - 1);
  const int seg = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * CC;
  const int first = A.seg_first[seg], count = A.seg_count[seg];
  const int g = h / (A.H / A.G), dp = A.dp, dv = A.dv;
  const bool folds = warp < kWarps;
  const int cl = (warp % kWarps) * CW + grp * NC;     // the group's first column, in the CTA
  float* sbase = A.state + (((int64_t)A.slot[first] * A.H + h) * dv) * dp;
  float4 S[NC][DR4];
  if (folds) {
    const bool fresh = A.pos[first] == 0;
#pragma unroll
    for (int s = 0; s < NC; ++s) {
      const int c = c0 + cl + (s ^ cb);
#pragma unroll
      for (int r = 0; r < DR4; ++r) {
        const int i = 4 * (p + LPC * r);
        S[s][r] = (!fresh && c < dv && i < dp) ? *reinterpret_cast<const float4*>(sbase + (int64_t)c * dp + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    }
  }
  if (dp < D)   // the key entries beyond dp are never staged: zeros in all buffers
    for (int i = tid; i < 3 * TS * (D - dp); i += 256) {
      const int j = i / (D - dp), e = dp + i - j * (D - dp);
      qs[j * D + e] = ks[j * D + e] = 0.f;
    }
  const int stages = (count + TS - 1) / TS;
  // iteration i: rows of stage i + 2 are fetched, scalars of stage i + 1 made, stage i folded in
  for (int it = -2; it < stages; ++it) {
    if (warp >= kWarps + 2) {
      if (it + 2 < stages) {
        const int b = (it + 2) % 3;
        stage_tokens<TS, CC>(A, first, count, (it + 2) * TS, g, h, c0, qs + b * TS * D, ks + b * TS * D, D, vs + b * TS * CC, gb + b * TS * 2,
                             tid - (kWarps + 2) * 32, 64);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
      }
    } else if (warp >= kWarps) {
      if (it >= -1 && it + 1 < stages) {
        const int b = (it + 1) % 3, blk = warp - kWarps;
        if ((it + 1) * TS + blk * kB8 < count)
          block_scalars<D>(ks + (b * TS + blk * kB8) * D, qs + (b * TS + blk * kB8) * D, gb + (b * TS + blk * kB8) * 2,
                           rec + (((it + 1) & 1) * TS + blk * kB8) * kRec, scratch + blk * 128);
      }
    } else if (it >= 0) {
      const int b = it % 3, t0 = it * TS;
      const float* kb = ks + b * TS * D;
      const float* qb = qs + b * TS * D;
      float* uw = us + cl * 8;
      const int nblk = (min(TS, count - t0) + kB8 - 1) / kB8;
      for (int blk = 0; blk < nblk; ++blk) {
        float a[kB8][NC], o[kB8][NC];
#pragma unroll
        for (int j = 0; j < kB8; ++j) {
          const int row = (blk * kB8 + (j ^ tb)) * D + 4 * p;
#pragma unroll
          for (int s = 0; s < NC; ++s) a[j][s] = o[j][s] = 0.f;
#pragma unroll
          for (int r = 0; r < DR4; ++r) {
            const float4 k = *reinterpret_cast<const float4*>(kb + row + 4 * LPC * r), q = *reinterpret_cast<const float4*>(qb + row + 4 * LPC * r);
#pragma unroll
            for (int s = 0; s < NC; ++s) a[j][s] = dot4(S[s][r], k, a[j][s]), o[j][s] = dot4(S[s][r], q, o[j][s]);
          }
        }
        const float* rc = rec + ((it & 1) * TS + blk * kB8 + tb) * kRec;
        const float4 r0 = *reinterpret_cast<const float4*>(rc);
        float T[kB8], C[kB8];
#pragma unroll
        for (int s = 0; s < kB8; s += 4) {
          *reinterpret_cast<float4*>(T + s) = *reinterpret_cast<const float4*>(rc + 4 + s);
          *reinterpret_cast<float4*>(C + s) = *reinterpret_cast<const float4*>(rc + 12 + s);
        }
        const float v = vs[(b * TS + blk * kB8 + tb) * CC + cl + cb];
#pragma unroll
        for (int half = kB8 / 2; half > 0; half >>= 1)
#pragma unroll
          for (int j = 0; j < half; ++j)
#pragma unroll
            for (int s = 0; s < NC; ++s) {
              a[j][s] += __shfl_xor_sync(0xffffffffu, a[j + half][s], half);
              o[j][s] += __shfl_xor_sync(0xffffffffu, o[j + half][s], half);
            }
#pragma unroll
        for (int half = NC / 2; half > 0; half >>= 1)
#pragma unroll
          for (int s = 0; s < half; ++s) {
            a[0][s] += __shfl_xor_sync(0xffffffffu, a[0][s + half], 8 * half);
            o[0][s] += __shfl_xor_sync(0xffffffffu, o[0][s + half], 8 * half);
          }
        const float w = r0.y * v - r0.x * a[0][0];
        float u = w, u2 = 0.f;
#pragma unroll
        for (int s = 1; s < kB8; ++s) {
          const float ws = __shfl_xor_sync(0xffffffffu, w, s);
          if (s & 1) u2 = fmaf(T[s], ws, u2);
          else u = fmaf(T[s], ws, u);
        }
        u += u2;
        __syncwarp();             // the group has read the previous block's values
        uw[cb * 8 + tb] = r0.w * u;
        __syncwarp();
        float4 e[NC][2];
#pragma unroll
        for (int s = 0; s < NC; ++s) {
          e[s][0] = *reinterpret_cast<const float4*>(uw + (s ^ cb) * 8);
          e[s][1] = *reinterpret_cast<const float4*>(uw + (s ^ cb) * 8 + 4);
        }
        const float G = T[0];
#pragma unroll
        for (int s = 0; s < NC; ++s)
#pragma unroll
          for (int r = 0; r < DR4; ++r) S[s][r].x *= G, S[s][r].y *= G, S[s][r].z *= G, S[s][r].w *= G;
#pragma unroll
        for (int j = 0; j < kB8; ++j)
#pragma unroll
          for (int r = 0; r < DR4; ++r) {
            const float4 k = *reinterpret_cast<const float4*>(kb + (blk * kB8 + j) * D + 4 * p + 4 * LPC * r);
#pragma unroll
            for (int s = 0; s < NC; ++s) {
              const float4 es = e[s][j / 4];
              const float x = j % 4 == 0 ? es.x : j % 4 == 1 ? es.y : j % 4 == 2 ? es.z : es.w;
              S[s][r].x = fmaf(x, k.x, S[s][r].x), S[s][r].y = fmaf(x, k.y, S[s][r].y);
              S[s][r].z = fmaf(x, k.z, S[s][r].z), S[s][r].w = fmaf(x, k.w, S[s][r].w);
            }
          }
        float y = fmaf(C[0], u, r0.z * o[0][0]), y2 = 0.f;
#pragma unroll
        for (int s = 1; s < kB8; ++s) {
          const float x = __shfl_xor_sync(0xffffffffu, u, s);
          if (s & 1) y2 = fmaf(C[s], x, y2);
          else y = fmaf(C[s], x, y);
        }
        const int t = t0 + blk * kB8 + tb, c = c0 + cl + cb;
        if (t < count && c < dv) A.out[(int64_t)(first + t) * A.H * dv + (int64_t)h * dv + c] = y + y2;
      }
    }
    __syncthreads();
  }
  if (folds) {
#pragma unroll
    for (int s = 0; s < NC; ++s) {
      const int c = c0 + cl + (s ^ cb);
#pragma unroll
      for (int r = 0; r < DR4; ++r) {
        const int i = 4 * (p + LPC * r);
        if (c < dv && i < dp) *reinterpret_cast<float4*>(sbase + (int64_t)c * dp + i) = S[s][r];
      }
    }
  }
  save_conv_memory(A, first, count);
}

template <int DR4, int LPC>
int launch_block8(const DeltaArgs& A, int n_segments, cudaStream_t st) {
  constexpr int TS = 16, CW = (LPC / 8) * (32 / LPC), CC = kWarps * CW, D = LPC * DR4 * 4;
  constexpr size_t smem = ((size_t)6 * TS * D + 3 * TS * CC + 3 * TS * 2 + 2 * TS * kRec + kWarps * CW * 8 + (TS / kB8) * 128) * sizeof(float);
  static_assert(smem <= 200 * 1024, "");
  auto kern = delta_block8_kernel<DR4, LPC>;
  if (smem > 48 * 1024) {
    static bool set = false;   // per instantiation
    if (!set) {
      if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return AO_B200_ERR_CUDA;
      set = true;
    }
  }
  kern<<<dim3((unsigned)n_segments, (unsigned)A.H, (unsigned)((A.dv + CC - 1) / CC)), 256, smem, st>>>(A);
  return lm_launch_status();
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
// This form takes any sizes.
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

// The same with whole 16-byte pieces (sizes and rows in multiples of four): a lane holds P pieces of a unit (a head of up to
// 128 P entries, or 128 P value channels), the convolution's taps in registers, for rows_per_warp consecutive rows.
template <typename T, int TAPS, int P>
__global__ void __launch_bounds__(256) delta_prep_vec_kernel(const float* __restrict__ proj, int64_t ld, int64_t conv_off, int64_t a_off,
                                                             int64_t b_off, int64_t n, int rows_per_warp, int H, int G, int d, int dv,
                                                             const T* __restrict__ conv_w, const float* __restrict__ conv_state,
                                                             const int32_t* __restrict__ slot, const int32_t* __restrict__ pos,
                                                             const int32_t* __restrict__ back, const T* __restrict__ a_log,
                                                             const T* __restrict__ dt_bias, float unit_eps, float q_scale,
                                                             float* __restrict__ qk, float* __restrict__ v, float* __restrict__ gb) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int hv = H * dv, qkc = 2 * G * d, C = qkc + hv;
  const int vunits = (hv + 128 * P - 1) / (128 * P), gunits = (H + 31) / 32, units = 2 * G + vunits + gunits;
  const int un = blockIdx.y * 8 + warp;
  if (un >= units) return;
  const int64_t t0 = (int64_t)blockIdx.x * rows_per_warp, t1 = t0 + rows_per_warp < n ? t0 + rows_per_warp : n;
  if (un >= 2 * G + vunits) {
    const int h = (un - 2 * G - vunits) * 32 + lane;
    if (h >= H) return;
    const float bias = ldf(dt_bias + h), rate = expf(ldf(a_log + h));
    for (int64_t t = t0; t < t1; ++t) {
      const float z = proj[t * ld + a_off + h] + bias;
      const float soft = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
      gb[(t * H + h) * 2] = expf(-rate * soft);
      gb[(t * H + h) * 2 + 1] = 1.f / (1.f + expf(-proj[t * ld + b_off + h]));
    }
    return;
  }
  const bool head = un < 2 * G;
  const int c0 = head ? un * d : qkc + (un - 2 * G) * 128 * P, c1 = head ? c0 + d : min(C, c0 + 128 * P);
  float4 w[TAPS][P];
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
#pragma unroll
    for (int e = 0; e < P; ++e) {
      const int c = c0 + 4 * (lane + 32 * e);
      w[j][e] = c < c1 ? ld4(conv_w + (int64_t)j * C + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  for (int64_t t = t0; t < t1; ++t) {
    const int bk = back[t], ps = pos[t];
    const float* x = proj + t * ld + conv_off;
    float4 y[P];
#pragma unroll
    for (int e = 0; e < P; ++e) y[e] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int delta = TAPS - 1 - j;     // rows back in time: in the step, in the slot's memory, or in front of the start
      if (delta > bk && delta > ps) continue;
      const float* row = delta <= bk ? x - (int64_t)delta * ld : conv_state + ((int64_t)slot[t] * (TAPS - 1) + (TAPS - 1 - (delta - bk))) * C;
#pragma unroll
      for (int e = 0; e < P; ++e) {
        const int c = c0 + 4 * (lane + 32 * e);
        if (c < c1) {
          const float4 u = *reinterpret_cast<const float4*>(row + c);
          y[e].x = fmaf(w[j][e].x, u.x, y[e].x), y[e].y = fmaf(w[j][e].y, u.y, y[e].y);
          y[e].z = fmaf(w[j][e].z, u.z, y[e].z), y[e].w = fmaf(w[j][e].w, u.w, y[e].w);
        }
      }
    }
    auto silu = [](float z) { return __fdividef(z, 1.f + expf(-z)); };
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < P; ++e) {
      y[e].x = silu(y[e].x), y[e].y = silu(y[e].y), y[e].z = silu(y[e].z), y[e].w = silu(y[e].w);
      ss = dot4(y[e], y[e], ss);
    }
    float* dst = v + t * hv + (c0 - qkc);
    float k = 1.f;
    if (head) {
      k = (un < G ? q_scale : 1.f) / sqrtf(warp_sum(ss) + unit_eps);
      dst = qk + (t * 2 * G + un) * d;
    }
#pragma unroll
    for (int e = 0; e < P; ++e) {
      const int i = 4 * (lane + 32 * e);
      if (c0 + i < c1) *reinterpret_cast<float4*>(dst + i) = make_float4(y[e].x * k, y[e].y * k, y[e].z * k, y[e].w * k);
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
  const cudaStream_t st = lm_stream(stream);
  auto on = [](const void* p, size_t bytes) { return reinterpret_cast<uintptr_t>(p) % bytes == 0; };
  const bool vec = d % 4 == 0 && (H * dv) % 4 == 0 && ld % 4 == 0 && conv_off % 4 == 0 && d <= 256 && taps >= 2 && taps <= 4 && on(proj, 16) &&
                   on(conv_w, dt == AO_LM_BF16 ? 8 : 16) && on(conv_state, 16) && on(qk, 16) && on(v, 16);
  if (vec) {
    const int P = d <= 128 ? 1 : 2, units = 2 * G + (H * dv + 128 * P - 1) / (128 * P) + (H + 31) / 32;
    const int rows = n >= 512 ? 4 : 1;      // many rows: a warp keeps its taps for several of them
    const dim3 grid((unsigned)((n + rows - 1) / rows), (unsigned)((units + 7) / 8));
    LM_CHECK_ARG(grid.y <= 65535);
#define LM_PREP(TAPS, PP)                                                                                                             \
  delta_prep_vec_kernel<T, TAPS, PP><<<grid, 256, 0, st>>>(proj, ld, conv_off, a_off, b_off, n, rows, H, G, d, dv,                    \
                                                           static_cast<const T*>(conv_w), conv_state, slot, pos, back,                \
                                                           static_cast<const T*>(a_log), static_cast<const T*>(dt_bias), unit_eps,    \
                                                           q_scale, qk, v, gb)
    LM_DISPATCH(dt, {
      if (taps == 4 && P == 1) LM_PREP(4, 1);
      else if (taps == 4) LM_PREP(4, 2);
      else if (taps == 3 && P == 1) LM_PREP(3, 1);
      else if (taps == 3) LM_PREP(3, 2);
      else if (P == 1) LM_PREP(2, 1);
      else LM_PREP(2, 2);
    });
#undef LM_PREP
    return lm_launch_status();
  }
  const int units = 2 * G + (H * dv + 127) / 128 + (H + 31) / 32;
  const unsigned parts = (unsigned)((units + 7) / 8 > 64 ? 64 : (units + 7) / 8);
  LM_DISPATCH(dt, delta_prep_kernel<T><<<dim3((unsigned)n, parts), 256, 0, st>>>(
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
  LM_CHECK_ARG(reinterpret_cast<uintptr_t>(qk) % 16 == 0 && reinterpret_cast<uintptr_t>(state) % 16 == 0 && (block == 1 || block == 8));
  const DeltaArgs A{qk, v, gb, H, G, dp, dv, state, slot, pos, seg_first, seg_count, conv_x, ld_conv, channels, taps, conv_state, out};
  const cudaStream_t st = lm_stream(stream);
  if (block == 8) {
    if (dp <= 64) return launch_block8<1, 16>(A, n_segments, st);
    if (dp <= 128) return launch_block8<1, 32>(A, n_segments, st);
    if (dp <= 256) return launch_block8<2, 32>(A, n_segments, st);
    if (dp <= 512) return launch_delta<4, 32, 4, 8>(A, n_segments, st);
    if (dp <= 1024) return launch_delta<8, 32, 4, 8>(A, n_segments, st);
    return AO_B200_ERR_UNSUPPORTED;
  }
#define LM_DELTA(DR4, LPC) return launch_delta<DR4, LPC, 1, 4>(A, n_segments, st)
  if (dp <= 16) LM_DELTA(1, 4);
  if (dp <= 32) LM_DELTA(1, 8);
  if (dp <= 64) LM_DELTA(2, 8);
  if (dp <= 128) LM_DELTA(4, 8);
  if (dp <= 256) LM_DELTA(4, 16);
  if (dp <= 512) LM_DELTA(4, 32);
  if (dp <= 1024) LM_DELTA(8, 32);
#undef LM_DELTA
  return AO_B200_ERR_UNSUPPORTED;
}

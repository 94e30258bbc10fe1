// Latent attention whose queries also come from a latent, under a sliding window or over a full cache: what happens between its projections.
//     ao_lm_latent_low_prep     projection row -> normed query latent, normed key/value latent, rotated shared key part
//                               (_store: also into a cache that never wraps, which saves the append launch)
//     ao_lm_latent_query_prep   up-projected queries -> unrotated parts (head-major) and rotated parts
//     ao_lm_latent_query_fold   the same for few rows, with the key up-projection folded into the unrotated parts
//     ao_lm_latent_rows_gather  the rows a step's queries can see, contiguous per sequence: window rows that earlier steps
//                               left in the ring, then the step's own
//     ao_lm_latent_value_up     weighted latents of few rows -> heads, times the sigmoid of an element-wise gate
//     ao_lm_sigmoid_gate_rows   the gate alone, in place (many rows: a library product made the heads)
// The step's latents stay in step buffers until its attention has run (ao_lm_ring_append then stores them): a long portion
// would otherwise overwrite ring rows that its first queries still need.  Norms and angles are fp32.
#include "lm_common.cuh"

using namespace lm;

namespace {

template <bool VEC>
__device__ __forceinline__ float part_squares(const float* __restrict__ src, int count) {
  float ss = 0.f;
  if (VEC) {
    for (int i = threadIdx.x * 4; i < count; i += blockDim.x * 4) {
      const float4 v = ld4(src + i);
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
  } else {
    for (int i = threadIdx.x; i < count; i += blockDim.x) ss = fmaf(src[i], src[i], ss);
  }
  return ss;
}
// out (and also, unless it is null) = src * k * weight
template <typename T, bool VEC>
__device__ __forceinline__ void scale_part(const float* __restrict__ src, int count, float k, const T* __restrict__ weight, T* __restrict__ out,
                                           T* __restrict__ also) {
  if (VEC) {
    for (int i = threadIdx.x * 4; i < count; i += blockDim.x * 4) {
      float4 v = ld4(src + i);
      const float4 g = ld4(weight + i);
      v.x *= k * g.x, v.y *= k * g.y, v.z *= k * g.z, v.w *= k * g.w;
      st4(out + i, v);
      if (also) st4(also + i, v);
    }
  } else {
    for (int i = threadIdx.x; i < count; i += blockDim.x) {
      const float v = src[i] * k * ldf(weight + i);
      stf(out + i, v);
      if (also) stf(also + i, v);
    }
  }
}

// One CTA per row.  The two norms' sums meet in one reduction (the row is read again from L1 for the output).  With c_cache the
// latent and the rotated part also go to row pos[t] of the slot (a cache that never wraps).
template <typename T, bool VEC>
__global__ void latent_low_prep_kernel(const float* __restrict__ proj, int64_t ld, int64_t q_off, int Rq, int64_t kv_off, int R, int dr,
                                       const T* __restrict__ q_norm, const T* __restrict__ c_norm, float eps, int rot_dims,
                                       const float* __restrict__ inv_freq, float amp, const int32_t* __restrict__ pos,
                                       const int32_t* __restrict__ slot, int64_t S, T* __restrict__ cq, T* __restrict__ c, T* __restrict__ kr,
                                       T* __restrict__ c_cache, T* __restrict__ kr_cache) {
  __shared__ float2 sums[32];
  pdl_trigger();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const float* row = proj + t * ld;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const float* src = row + kv_off + R;
  const int half = rot_dims / 2;
  const int p = pos[t];
  const int64_t at = c_cache ? (int64_t)slot[t] * S + p : 0;
  float sq = warp_sum(part_squares<VEC>(row + q_off, Rq)), sc = warp_sum(part_squares<VEC>(row + kv_off, R));
  if (lane == 0) sums[warp] = make_float2(sq, sc);
  // the shared key part meanwhile
  T* dst = kr + t * dr;
  T* also = kr_cache ? kr_cache + at * dr : nullptr;
  for (int i = threadIdx.x; i < dr - half; i += blockDim.x) {
    if (i < half) {
      float sn, cs;
      sincosf((float)p * inv_freq[i], &sn, &cs);
      sn *= amp, cs *= amp;
      const float u = src[2 * i], v = src[2 * i + 1];
      const float a = u * cs - v * sn, b = v * cs + u * sn;
      stf(dst + 2 * i, a);
      stf(dst + 2 * i + 1, b);
      if (also) {
        stf(also + 2 * i, a);
        stf(also + 2 * i + 1, b);
      }
    } else {
      stf(dst + half + i, src[half + i]);     // coordinates from rot_dims on pass
      if (also) stf(also + half + i, src[half + i]);
    }
  }
  __syncthreads();
  const float2 mine = lane < nw ? sums[lane] : make_float2(0.f, 0.f);
  sq = warp_sum(mine.x), sc = warp_sum(mine.y);
  scale_part<T, VEC>(row + q_off, Rq, 1.f / sqrtf(sq / (float)Rq + eps), q_norm, cq + t * Rq, nullptr);
  scale_part<T, VEC>(row + kv_off, R, 1.f / sqrtf(sc / (float)R + eps), c_norm, c + t * R, c_cache ? c_cache + at * R : nullptr);
}

// q [n][H][dn + dr] -> qn[h][t][dn] in T, qr[t][h][dr] rotated, fp32.  A row may be shared by several CTAs.
template <typename T>
__global__ void latent_query_prep_kernel(const float* __restrict__ q, int64_t n, int H, int dn, int dr, int rot_dims,
                                         const float* __restrict__ inv_freq, float amp, const int32_t* __restrict__ pos,
                                         T* __restrict__ qn, float* __restrict__ qr) {
  const int64_t t = blockIdx.x;
  const int tid = blockIdx.y * blockDim.x + threadIdx.x, nth = gridDim.y * blockDim.x;
  const float* row = q + t * H * (dn + dr);
  for (int i = tid; i < H * dn; i += nth) {
    const int h = i / dn, e = i - h * dn;
    stf(qn + ((int64_t)h * n + t) * dn + e, row[h * (dn + dr) + e]);
  }
  const float p = (float)pos[t];
  const int half = rot_dims / 2, per = dr - half;
  for (int i = tid; i < H * per; i += nth) {
    const int h = i / per, e = i - h * per;
    const float* src = row + h * (dn + dr) + dn;
    float* dst = qr + (t * H + h) * dr;
    if (e < half) {
      float sn, cs;
      sincosf(p * inv_freq[e], &sn, &cs);
      sn *= amp, cs *= amp;
      const float u = src[2 * e], v = src[2 * e + 1];
      dst[2 * e] = u * cs - v * sn;
      dst[2 * e + 1] = v * cs + u * sn;
    } else {
      dst[half + e] = src[half + e];
    }
  }
}

// out row i = step row src[i] when src[i] >= 0, else ring row -1 - src[i] (slot * ring + position % ring)
template <typename T>
__global__ void latent_rows_gather_kernel(const int32_t* __restrict__ src, const T* __restrict__ c, const T* __restrict__ kr,
                                          const T* __restrict__ ring_c, const T* __restrict__ ring_kr, int R, int dr,
                                          T* __restrict__ out_c, T* __restrict__ out_kr) {
  const int64_t i = blockIdx.x;
  const int s = src[i];
  const int64_t r = s >= 0 ? s : -1 - (int64_t)s;
  const T* a = (s >= 0 ? c : ring_c) + r * R;
  const T* b = (s >= 0 ? kr : ring_kr) + r * dr;
  constexpr int kPer = 16 / (int)sizeof(T);
  const bool vec = R % kPer == 0 && reinterpret_cast<uintptr_t>(a) % 16 == 0 && reinterpret_cast<uintptr_t>(out_c) % 16 == 0;
  if (vec) {
    const uint4* a4 = reinterpret_cast<const uint4*>(a);
    uint4* o4 = reinterpret_cast<uint4*>(out_c + i * R);
    for (int e = threadIdx.x; e < R / kPer; e += blockDim.x) o4[e] = a4[e];
  } else {
    for (int e = threadIdx.x; e < R; e += blockDim.x) out_c[i * R + e] = a[e];
  }
  for (int e = threadIdx.x; e < dr; e += blockDim.x) out_kr[i * dr + e] = b[e];
}

// out[t][h dv + j] = sigmoid(gate[t][h dv + j]) * sum_r uv[h][j][r] * olat[t][h][r].  One CTA = one row x one head x kUpOut
// outputs; a warp makes four of them at a time from one pass over their weight rows.
constexpr int kUpWarps = 8, kUpPer = 4, kUpOut = kUpWarps * kUpPer, kUpHold = 2;   // kUpHold: 16-byte pieces of a row per lane
template <typename T>
__global__ void __launch_bounds__(kUpWarps * 32) latent_value_up_kernel(const T* __restrict__ olat, const T* __restrict__ uv, int H, int R,
                                                                        int dv, const float* __restrict__ gate, int64_t ld_gate, bool vec,
                                                                        T* __restrict__ out, int64_t ld_out) {
  extern __shared__ __align__(16) float xs[];
  constexpr int kPer = 16 / (int)sizeof(T);
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t t = blockIdx.z;
  const int j0 = blockIdx.x * kUpOut + warp * kUpPer, nr = min(kUpPer, dv - j0);
  const T* rows[kUpPer];
#pragma unroll
  for (int i = 0; i < kUpPer; ++i) rows[i] = uv + ((int64_t)h * dv + (i < nr ? j0 + i : 0)) * R;
  const int pieces = vec ? R / kPer : 0;
  uint4 w[kUpPer][kUpHold];
  pdl_trigger();
#pragma unroll
  for (int i = 0; i < kUpPer; ++i)        // the weights depend on nothing: they travel while the launch in front finishes
#pragma unroll
    for (int u = 0; u < kUpHold; ++u)
      w[i][u] = lane + 32 * u < pieces ? __ldg(reinterpret_cast<const uint4*>(rows[i]) + lane + 32 * u) : make_uint4(0, 0, 0, 0);
  pdl_wait();
  const int64_t col = (int64_t)h * dv + j0 + lane;
  const float logit = gate && lane < nr ? gate[t * ld_gate + col] : 0.f;
  stage_f32(olat + (t * H + h) * R, xs, R);
  __syncthreads();
  if (nr <= 0) return;
  float acc[kUpPer] = {0.f, 0.f, 0.f, 0.f};
  auto use = [&](int i, const uint4& v, int piece) {
    float f[kPer];
    unpack16(v, f, static_cast<const T*>(nullptr));
#pragma unroll
    for (int e = 0; e < kPer; ++e) acc[i] = fmaf(f[e], xs[piece * kPer + e], acc[i]);
  };
#pragma unroll
  for (int u = 0; u < kUpHold; ++u)
    if (lane + 32 * u < pieces)
#pragma unroll
      for (int i = 0; i < kUpPer; ++i) use(i, w[i][u], lane + 32 * u);
  for (int piece = lane + 32 * kUpHold; piece < pieces; piece += 32)
#pragma unroll
    for (int i = 0; i < kUpPer; ++i) use(i, __ldg(reinterpret_cast<const uint4*>(rows[i]) + piece), piece);
  if (!vec)
    for (int r = lane; r < R; r += 32)
#pragma unroll
      for (int i = 0; i < kUpPer; ++i) acc[i] = fmaf(ldf(rows[i] + r), xs[r], acc[i]);
#pragma unroll
  for (int i = 0; i < kUpPer; ++i) acc[i] = warp_sum(acc[i]);
  if (lane < nr) {
    float v = acc[0];
#pragma unroll
    for (int i = 1; i < kUpPer; ++i)
      if (lane == i) v = acc[i];
    if (gate) v = v / (1.f + expf(-logit));
    stf(out + t * ld_out + col, v);
  }
}

// The folded form's way in, for few rows: q fp32 [n][H][dn + dr] -> qa[h][t][r] = sum_d uk[h][d][r] * q[t][h][d] (fp32) and
// qr[t][h][:] = the rotated part.  One CTA = one head x kFoldCols latent coordinates x one row: a thread owns eight coordinates
// and every kFoldParts-th d; the partial sums meet in shared memory.
constexpr int kFoldCols = 64, kFoldParts = 32, kFoldHold = 4;     // kFoldHold: weights per thread that travel before the wait
__global__ void __launch_bounds__(kFoldCols / 8 * kFoldParts) latent_query_fold_kernel(
    const float* __restrict__ q, const __nv_bfloat16* __restrict__ uk, int64_t n, int H, int dn, int dr, int R, int rot_dims,
    const float* __restrict__ inv_freq, float amp, const int32_t* __restrict__ pos, float* __restrict__ qa, float* __restrict__ qr) {
  __shared__ float part[kFoldParts][kFoldCols + 1];
  const int h = blockIdx.y, c8 = threadIdx.x % (kFoldCols / 8), dp = threadIdx.x / (kFoldCols / 8);
  const int64_t t = blockIdx.z;
  const int r0 = blockIdx.x * kFoldCols + c8 * 8;
  const __nv_bfloat16* w0 = uk + (int64_t)h * dn * R + min(r0, R - 8);
  uint4 w[kFoldHold];
  pdl_trigger();
#pragma unroll
  for (int u = 0; u < kFoldHold; ++u) {
    const int d = dp + u * kFoldParts;
    w[u] = d < dn ? __ldg(reinterpret_cast<const uint4*>(w0 + (int64_t)d * R)) : make_uint4(0, 0, 0, 0);
  }
  pdl_wait();
  const float* row = q + (t * H + h) * (dn + dr);
  float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  auto use = [&](const uint4& v, float x) {
    float f[8];
    unpack16(v, f, static_cast<const __nv_bfloat16*>(nullptr));
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = fmaf(f[e], x, acc[e]);
  };
#pragma unroll
  for (int u = 0; u < kFoldHold; ++u)
    if (dp + u * kFoldParts < dn) use(w[u], row[dp + u * kFoldParts]);
  for (int d = dp + kFoldHold * kFoldParts; d < dn; d += kFoldParts) use(__ldg(reinterpret_cast<const uint4*>(w0 + (int64_t)d * R)), row[d]);
#pragma unroll
  for (int e = 0; e < 8; ++e) part[dp][c8 * 8 + e] = acc[e];
  if (blockIdx.x == 0) {        // this head's rotated part
    const float p = (float)pos[t];
    const int half = rot_dims / 2;
    float* dst = qr + (t * H + h) * dr;
    for (int i = threadIdx.x; i < dr - half; i += blockDim.x) {
      const float* src = row + dn;
      if (i < half) {
        float sn, cs;
        sincosf(p * inv_freq[i], &sn, &cs);
        sn *= amp, cs *= amp;
        const float u = src[2 * i], v = src[2 * i + 1];
        dst[2 * i] = u * cs - v * sn;
        dst[2 * i + 1] = v * cs + u * sn;
      } else {
        dst[half + i] = src[half + i];
      }
    }
  }
  __syncthreads();
  for (int c = threadIdx.x; c < kFoldCols; c += blockDim.x) {
    const int r = blockIdx.x * kFoldCols + c;
    if (r >= R) break;
    float s = 0.f;
#pragma unroll
    for (int d = 0; d < kFoldParts; ++d) s += part[d][c];
    qa[((int64_t)h * n + t) * R + r] = s;
  }
}

template <typename T>
__global__ void sigmoid_gate_rows_kernel(const float* __restrict__ gate, int64_t ld_gate, int64_t cols, T* y, int64_t ld) {
  const int64_t t = blockIdx.x;
  for (int64_t c = (int64_t)blockIdx.y * blockDim.x + threadIdx.x; c < cols; c += (int64_t)gridDim.y * blockDim.x)
    stf(y + t * ld + c, ldf(y + t * ld + c) / (1.f + expf(-gate[t * ld_gate + c])));
}

}  // namespace

extern "C" int ao_lm_latent_low_prep_store(const float* proj, int64_t ld, int64_t n, int64_t q_off, int Rq, int64_t kv_off, int R, int dr,
                                           const void* q_norm, const void* c_norm, int dt, float eps, int rot_dims, const float* inv_freq,
                                           float amp, const int32_t* pos, const int32_t* slot, int64_t S, void* cq, void* c, void* kr,
                                           void* c_cache, void* kr_cache, void* stream) {
  LM_CHECK_ARG(proj && q_norm && c_norm && pos && cq && c && (kr || dr == 0) && n > 0 && Rq > 0 && R > 0 && dr >= 0);
  LM_CHECK_ARG(rot_dims >= 0 && rot_dims <= dr && rot_dims % 2 == 0 && (rot_dims == 0 || inv_freq));
  LM_CHECK_ARG(!c_cache || (slot && S > 0 && (kr_cache || dr == 0)));
  LM_DISPATCH(dt, {
    auto on = [](const void* p, size_t bytes) { return reinterpret_cast<uintptr_t>(p) % bytes == 0; };
    const size_t four = 4 * sizeof(T);
    const bool vec = ld % 4 == 0 && q_off % 4 == 0 && kv_off % 4 == 0 && Rq % 4 == 0 && R % 4 == 0 && on(proj, 16) && on(q_norm, four) &&
                     on(c_norm, four) && on(cq, four) && on(c, four) && on(c_cache, four);
    auto kern = vec ? latent_low_prep_kernel<T, true> : latent_low_prep_kernel<T, false>;
    return lm_launch_early(kern, dim3((unsigned)n), dim3(n < 296 && !vec ? 512 : n < 296 ? 256 : 128), 0, lm_stream(stream), proj, ld, q_off, Rq,
                           kv_off, R, dr, static_cast<const T*>(q_norm), static_cast<const T*>(c_norm), eps, rot_dims, inv_freq, amp, pos, slot, S,
                           static_cast<T*>(cq), static_cast<T*>(c), static_cast<T*>(kr), static_cast<T*>(c_cache), static_cast<T*>(kr_cache));
  });
  return AO_B200_OK;
}

extern "C" int ao_lm_latent_low_prep(const float* proj, int64_t ld, int64_t n, int64_t q_off, int Rq, int64_t kv_off, int R, int dr,
                                     const void* q_norm, const void* c_norm, int dt, float eps, int rot_dims, const float* inv_freq,
                                     float amp, const int32_t* pos, void* cq, void* c, void* kr, void* stream) {
  return ao_lm_latent_low_prep_store(proj, ld, n, q_off, Rq, kv_off, R, dr, q_norm, c_norm, dt, eps, rot_dims, inv_freq, amp, pos, nullptr, 0,
                                     cq, c, kr, nullptr, nullptr, stream);
}

extern "C" int ao_lm_latent_query_prep(const float* q, int64_t n, int H, int dn, int dr, int dt, int rot_dims, const float* inv_freq,
                                       float amp, const int32_t* pos, void* qn, float* qr, void* stream) {
  LM_CHECK_ARG(q && pos && qn && (qr || dr == 0) && n > 0 && H > 0 && dn > 0 && dr >= 0);
  LM_CHECK_ARG(rot_dims >= 0 && rot_dims <= dr && rot_dims % 2 == 0 && (rot_dims == 0 || inv_freq));
  const int64_t items = (int64_t)H * (dn + dr);
  const int64_t room = (592 + n - 1) / n, want = (items + 511) / 512;
  const unsigned parts = n < 296 ? (unsigned)(want > room ? room : want < 1 ? 1 : want) : 1u;
  LM_DISPATCH(dt, latent_query_prep_kernel<T><<<dim3((unsigned)n, parts), 256, 0, lm_stream(stream)>>>(
                      q, n, H, dn, dr, rot_dims, inv_freq, amp, pos, static_cast<T*>(qn), qr));
  return lm_launch_status();
}

extern "C" int ao_lm_latent_rows_gather(const int32_t* src, int64_t rows, const void* c, const void* kr, const void* ring_c,
                                        const void* ring_kr, int dt, int R, int dr, void* out_c, void* out_kr, void* stream) {
  LM_CHECK_ARG(src && rows > 0 && c && ring_c && out_c && R > 0 && dr >= 0 && (dr == 0 || (kr && ring_kr && out_kr)));
  LM_DISPATCH(dt, latent_rows_gather_kernel<T><<<(unsigned)rows, 64, 0, lm_stream(stream)>>>(
                      src, static_cast<const T*>(c), static_cast<const T*>(kr), static_cast<const T*>(ring_c),
                      static_cast<const T*>(ring_kr), R, dr, static_cast<T*>(out_c), static_cast<T*>(out_kr)));
  return lm_launch_status();
}

extern "C" int ao_lm_latent_value_up(const void* olat, const void* uv, int dt, int64_t n, int H, int R, int dv, const float* gate,
                                     int64_t ld_gate, void* out, int64_t ld_out, void* stream) {
  LM_CHECK_ARG(olat && uv && out && n > 0 && n <= 65535 && H > 0 && H <= 65535 && R > 0 && dv > 0 && ld_out >= (int64_t)H * dv &&
               (!gate || ld_gate >= (int64_t)H * dv));
  if ((size_t)R * sizeof(float) > 48 * 1024) return AO_B200_ERR_UNSUPPORTED;
  LM_DISPATCH(dt, return lm_launch_early(latent_value_up_kernel<T>, dim3((unsigned)((dv + kUpOut - 1) / kUpOut), (unsigned)H, (unsigned)n),
                                         dim3(kUpWarps * 32), (size_t)R * sizeof(float), lm_stream(stream), static_cast<const T*>(olat),
                                         static_cast<const T*>(uv), H, R, dv, gate, ld_gate, rows_vectorizable<T>(uv, R), static_cast<T*>(out),
                                         ld_out));
  return AO_B200_OK;
}

extern "C" int ao_lm_latent_query_fold(const float* q, const void* uk, int dt, int64_t n, int H, int dn, int dr, int R, int rot_dims,
                                       const float* inv_freq, float amp, const int32_t* pos, float* qa, float* qr, void* stream) {
  LM_CHECK_ARG(q && uk && pos && qa && (qr || dr == 0) && n > 0 && n <= 65535 && H > 0 && H <= 65535 && dn > 0 && dr >= 0 && R > 0);
  LM_CHECK_ARG(rot_dims >= 0 && rot_dims <= dr && rot_dims % 2 == 0 && (rot_dims == 0 || inv_freq));
  if (dt != AO_LM_BF16 || R % 8 || reinterpret_cast<uintptr_t>(uk) % 16) return AO_B200_ERR_UNSUPPORTED;
  return lm_launch_early(latent_query_fold_kernel, dim3((unsigned)((R + kFoldCols - 1) / kFoldCols), (unsigned)H, (unsigned)n),
                         dim3(kFoldCols / 8 * kFoldParts), 0, lm_stream(stream), q, static_cast<const __nv_bfloat16*>(uk), n, H, dn, dr, R,
                         rot_dims, inv_freq, amp, pos, qa, qr);
}

extern "C" int ao_lm_sigmoid_gate_rows(const float* gate, int64_t ld_gate, int64_t n, int64_t cols, void* y, int64_t ld, int dt,
                                       void* stream) {
  LM_CHECK_ARG(gate && y && n > 0 && cols > 0 && ld >= cols && ld_gate >= cols);
  int64_t parts = (cols + 511) / 512;
  if (parts > 64) parts = 64;
  LM_DISPATCH(dt, sigmoid_gate_rows_kernel<T><<<dim3((unsigned)n, (unsigned)parts), 256, 0, lm_stream(stream)>>>(
                      gate, ld_gate, cols, static_cast<T*>(y), ld));
  return lm_launch_status();
}

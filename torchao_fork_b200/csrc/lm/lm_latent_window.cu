// Latent attention whose queries also come from a latent, under a sliding window: what happens between its projections.
//     ao_lm_latent_low_prep     projection row -> normed query latent, normed key/value latent, rotated shared key part
//     ao_lm_latent_query_prep   up-projected queries -> unrotated parts (head-major) and rotated parts
//     ao_lm_latent_rows_gather  the rows a step's queries can see, contiguous per sequence: window rows that earlier steps
//                               left in the ring, then the step's own
// The step's latents stay in step buffers until its attention has run (ao_lm_ring_append then stores them): a long portion
// would otherwise overwrite ring rows that its first queries still need.  Norms and angles are fp32.
#include "lm_common.cuh"

using namespace lm;

namespace {

// out[0 .. count) = src / sqrt(mean(src^2) + eps) * weight by the whole block
template <typename T>
__device__ __forceinline__ void norm_part(const float* __restrict__ src, int count, const T* __restrict__ weight, float eps,
                                          T* __restrict__ out, float* scratch) {
  float ss = 0.f;
  for (int i = threadIdx.x; i < count; i += blockDim.x) ss = fmaf(src[i], src[i], ss);
  const float k = 1.f / sqrtf(block_sum(ss, scratch) / (float)count + eps);
  for (int i = threadIdx.x; i < count; i += blockDim.x) stf(out + i, src[i] * k * ldf(weight + i));
}

template <typename T>
__global__ void latent_low_prep_kernel(const float* __restrict__ proj, int64_t ld, int64_t q_off, int Rq, int64_t kv_off, int R, int dr,
                                       const T* __restrict__ q_norm, const T* __restrict__ c_norm, float eps, int rot_dims,
                                       const float* __restrict__ inv_freq, float amp, const int32_t* __restrict__ pos,
                                       T* __restrict__ cq, T* __restrict__ c, T* __restrict__ kr) {
  __shared__ float scratch[33];
  const int64_t t = blockIdx.x;
  const float* row = proj + t * ld;
  norm_part(row + q_off, Rq, q_norm, eps, cq + t * Rq, scratch);
  norm_part(row + kv_off, R, c_norm, eps, c + t * R, scratch);
  const float* src = row + kv_off + R;
  T* dst = kr + t * dr;
  const float p = (float)pos[t];
  const int half = rot_dims / 2;
  for (int i = threadIdx.x; i < dr - half; i += blockDim.x) {
    if (i < half) {
      float sn, cs;
      sincosf(p * inv_freq[i], &sn, &cs);
      sn *= amp, cs *= amp;
      const float u = src[2 * i], v = src[2 * i + 1];
      stf(dst + 2 * i, u * cs - v * sn);
      stf(dst + 2 * i + 1, v * cs + u * sn);
    } else {
      stf(dst + half + i, src[half + i]);     // coordinates from rot_dims on pass
    }
  }
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

}  // namespace

extern "C" int ao_lm_latent_low_prep(const float* proj, int64_t ld, int64_t n, int64_t q_off, int Rq, int64_t kv_off, int R, int dr,
                                     const void* q_norm, const void* c_norm, int dt, float eps, int rot_dims, const float* inv_freq,
                                     float amp, const int32_t* pos, void* cq, void* c, void* kr, void* stream) {
  LM_CHECK_ARG(proj && q_norm && c_norm && pos && cq && c && (kr || dr == 0) && n > 0 && Rq > 0 && R > 0 && dr >= 0);
  LM_CHECK_ARG(rot_dims >= 0 && rot_dims <= dr && rot_dims % 2 == 0 && (rot_dims == 0 || inv_freq));
  LM_DISPATCH(dt, latent_low_prep_kernel<T><<<(unsigned)n, n < 296 ? 512 : 128, 0, lm_stream(stream)>>>(
                      proj, ld, q_off, Rq, kv_off, R, dr, static_cast<const T*>(q_norm), static_cast<const T*>(c_norm), eps, rot_dims,
                      inv_freq, amp, pos, static_cast<T*>(cq), static_cast<T*>(c), static_cast<T*>(kr)));
  return lm_launch_status();
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

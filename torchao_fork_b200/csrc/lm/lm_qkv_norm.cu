// Projection row -> what softmax attention reads, for designs that norm every query and key head: biases, RMS norm per head with
// one weight for all heads, rotation of the first coordinates, values in the storage type.  One warp per head; a row's angles
// are computed once per CTA.  When every sequence of the step brings one row (decoding), the keys and values also go straight
// into the ring: the row they replace is the one that has just left the window, so no append launch follows.
#include "lm_common.cuh"

using namespace lm;

namespace {

constexpr int kWarps = 8;

struct QkvArgs {
  const float* proj;
  int64_t ld, q_off, k_off, v_off;
  const void *q_bias, *k_bias, *v_bias, *q_weight, *k_weight;
  const int32_t *pos, *slot;
  const float* inv_freq;
  int rot_dims, pairing;
  float amp, eps;
  int H, G, d, v_width;
  float* qn;
  void *kn, *vn, *ring_k, *ring_v;
  int ring;
};

// VEC: d, rot_dims / 2 and v_width are multiples of four, every row starts on a 16-byte boundary, pairs are (i, i + rot_dims / 2)
template <typename T, bool VEC>
__global__ void __launch_bounds__(kWarps * 32) qkv_norm_rotary_kernel(QkvArgs a) {
  extern __shared__ __align__(16) float sm[];
  const int d = a.d, half = a.rot_dims / 2, dp = (d + 3) & ~3, hp = (half + 3) & ~3;
  float *cs = sm, *sn = sm + hp;                                    // cosines and sines of the row's pairs
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* buf = sm + 2 * hp + (size_t)warp * dp;                     // this warp's head, normed
  pdl_trigger();
  pdl_wait();
  const int64_t t = blockIdx.x;
  const int p = a.pos[t];
  const float* row = a.proj + t * a.ld;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf((float)p * a.inv_freq[i], &s, &c);
    cs[i] = c * a.amp, sn[i] = s * a.amp;
  }
  __syncthreads();
  const int64_t ring_row = a.ring_k ? (int64_t)a.slot[t] * a.ring + p % a.ring : 0;
  for (int hd = blockIdx.y * kWarps + warp; hd < a.H + a.G; hd += gridDim.y * kWarps) {
    const bool is_q = hd < a.H;
    const int64_t ho = (int64_t)(is_q ? hd : hd - a.H) * d;
    const float* src = row + (is_q ? a.q_off : a.k_off) + ho;
    const T* bias = static_cast<const T*>(is_q ? a.q_bias : a.k_bias);
    const T* weight = static_cast<const T*>(is_q ? a.q_weight : a.k_weight);
    float ss = 0.f;
    if (VEC) {
      for (int c = lane * 4; c < d; c += 128) {
        float4 v = ld4(src + c);
        if (bias) {
          const float4 b = ld4(bias + ho + c);
          v.x += b.x, v.y += b.y, v.z += b.z, v.w += b.w;
        }
        ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        if (weight) {
          const float4 g = ld4(weight + c);
          v.x *= g.x, v.y *= g.y, v.z *= g.z, v.w *= g.w;
        }
        st4(buf + c, v);
      }
    } else {
      for (int c = lane; c < d; c += 32) {
        float v = src[c] + (bias ? ldf(bias + ho + c) : 0.f);
        ss = fmaf(v, v, ss);
        buf[c] = weight ? v * ldf(weight + c) : v;
      }
    }
    const float k = weight ? 1.f / sqrtf(warp_sum(ss) / (float)d + a.eps) : 1.f;
    __syncwarp();
    float* qd = a.qn + t * a.H * d + ho;
    T* kd = static_cast<T*>(a.kn) + t * a.G * d + ho;
    T* rd = a.ring_k ? static_cast<T*>(a.ring_k) + ring_row * a.G * d + ho : nullptr;
    if (VEC) {
      for (int c = lane * 4; c < d; c += 128) {
        const float4 v = ld4(buf + c);
        float4 r = v;
        if (c < 2 * half) {
          const bool lo = c < half;
          const int i = lo ? c : c - half;
          const float4 o = ld4(buf + (lo ? c + half : c - half)), cc = ld4(cs + i);
          float4 s = ld4(sn + i);
          if (lo) s.x = -s.x, s.y = -s.y, s.z = -s.z, s.w = -s.w;
          r.x = v.x * cc.x + o.x * s.x, r.y = v.y * cc.y + o.y * s.y, r.z = v.z * cc.z + o.z * s.z, r.w = v.w * cc.w + o.w * s.w;
        }
        r.x *= k, r.y *= k, r.z *= k, r.w *= k;
        if (is_q) {
          st4(qd + c, r);
        } else {
          st4(kd + c, r);
          if (rd) st4(rd + c, r);
        }
      }
    } else {
      for (int c = lane; c < d; c += 32) {
        float r = buf[c];
        if (c < 2 * half) {
          const bool lo = a.pairing ? c < half : (c & 1) == 0;
          const int i = a.pairing ? (lo ? c : c - half) : c / 2, o = a.pairing ? (lo ? c + half : c - half) : c ^ 1;
          r = r * cs[i] + buf[o] * (lo ? -sn[i] : sn[i]);
        }
        r *= k;
        if (is_q) {
          qd[c] = r;
        } else {
          stf(kd + c, r);
          if (rd) stf(rd + c, r);
        }
      }
    }
    __syncwarp();
  }
  const T* v_bias = static_cast<const T*>(a.v_bias);
  T* vd = static_cast<T*>(a.vn) + t * a.v_width;
  T* rv = a.ring_v ? static_cast<T*>(a.ring_v) + ring_row * a.v_width : nullptr;
  const int tid = blockIdx.y * blockDim.x + threadIdx.x, nth = gridDim.y * blockDim.x;
  if (VEC) {
    for (int c = tid * 4; c < a.v_width; c += nth * 4) {
      float4 v = ld4(row + a.v_off + c);
      if (v_bias) {
        const float4 b = ld4(v_bias + c);
        v.x += b.x, v.y += b.y, v.z += b.z, v.w += b.w;
      }
      st4(vd + c, v);
      if (rv) st4(rv + c, v);
    }
  } else {
    for (int c = tid; c < a.v_width; c += nth) {
      const float v = row[a.v_off + c] + (v_bias ? ldf(v_bias + c) : 0.f);
      stf(vd + c, v);
      if (rv) stf(rv + c, v);
    }
  }
}

inline bool on(const void* p, size_t bytes) { return reinterpret_cast<uintptr_t>(p) % bytes == 0; }

}  // namespace

extern "C" int ao_lm_qkv_norm_rotary_prep(const float* proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, const void* q_bias,
                                          const void* k_bias, const void* v_bias, const void* q_weight, const void* k_weight, float eps,
                                          const int32_t* pos, const float* inv_freq, int rot_dims, int pairing, float amp, int64_t n, int H,
                                          int G, int d, int v_width, int dt, float* qn, void* kn, void* vn, const int32_t* slot, int ring,
                                          void* ring_k, void* ring_v, void* stream) {
  LM_CHECK_ARG(proj && pos && qn && kn && vn && n > 0 && H > 0 && G > 0 && d > 0 && v_width > 0);
  LM_CHECK_ARG(rot_dims >= 0 && rot_dims <= d && rot_dims % 2 == 0 && (rot_dims == 0 || inv_freq) && (pairing == 0 || pairing == 1));
  LM_CHECK_ARG((!ring_k && !ring_v) || (ring_k && ring_v && slot && ring > 0));
  const QkvArgs a{proj, ld, q_off, k_off, v_off, q_bias, k_bias, v_bias, q_weight, k_weight, pos, slot, inv_freq, rot_dims, pairing, amp, eps,
                  H, G, d, v_width, qn, kn, vn, ring_k, ring_v, ring};
  const int dp = (d + 3) & ~3, hp = (rot_dims / 2 + 3) & ~3;
  const size_t smem = (2 * (size_t)hp + (size_t)kWarps * dp) * sizeof(float);
  if (smem > 48 * 1024) return AO_B200_ERR_UNSUPPORTED;
  // few rows (decoded tokens): a row's heads are shared out over several CTAs
  const int64_t rounds = (H + G + kWarps - 1) / kWarps, room = (592 + n - 1) / n;
  const unsigned parts = (unsigned)(n >= 296 ? 1 : rounds < room ? rounds : room);
  LM_DISPATCH(dt, {
    const size_t four = 4 * sizeof(T);
    const bool vec = pairing == 1 && d % 4 == 0 && (rot_dims / 2) % 4 == 0 && v_width % 4 == 0 && ld % 4 == 0 && q_off % 4 == 0 &&
                     k_off % 4 == 0 && v_off % 4 == 0 && on(proj, 16) && on(qn, 16) && on(kn, four) && on(vn, four) && on(ring_k, four) &&
                     on(ring_v, four) && on(q_bias, four) && on(k_bias, four) && on(v_bias, four) && on(q_weight, four) && on(k_weight, four);
    auto kern = vec ? qkv_norm_rotary_kernel<T, true> : qkv_norm_rotary_kernel<T, false>;
    return lm_launch_early(kern, dim3((unsigned)n, parts), dim3(kWarps * 32), smem, lm_stream(stream), a);
  });
  return AO_B200_OK;
}

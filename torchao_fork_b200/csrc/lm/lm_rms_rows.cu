// Row kernels of designs with a plain pre-norm RMS residual in fp32: scaled embedding gather, residual add fused with the
// next RMS norm, and the xIELU activation between two projections.  Every kernel reads and writes rows inside wider rows
// (row strides), so that several sublayers can share one projection and one output product.
#include "lm_common.cuh"

using namespace lm;

namespace {

template <typename T>
__global__ void embed_scaled_kernel(const T* __restrict__ table, const int64_t* __restrict__ tok, int64_t W, float scale,
                                    float* __restrict__ x) {
  const int64_t t = blockIdx.x;
  const T* row = table + tok[t] * W;
  for (int64_t w = threadIdx.x; w < W; w += blockDim.x) x[t * W + w] = ldf(row + w) * scale;
}

// x[r] += y[r];  out[i] = x[r] / sqrt(mean(x[r]^2) + eps) * weight,  r = rows ? rows[i] : i.  One CTA per row; the row stays
// on chip between the sum of squares and the output.  VEC: four values per access.
template <typename T, bool VEC>
__global__ void add_rms_norm_kernel(float* x, const float* __restrict__ y, const int32_t* __restrict__ rows, int64_t W,
                                    const T* __restrict__ weight, float eps, T* __restrict__ out) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[33];
  const int64_t i = blockIdx.x, r = rows ? (int64_t)rows[i] : i;
  float* xr = x + r * W;
  const float* yr = y ? y + r * W : nullptr;
  float ss = 0.f;
  if (VEC) {
    for (int64_t w = (int64_t)threadIdx.x * 4; w < W; w += (int64_t)blockDim.x * 4) {
      float4 v = ld4(xr + w);
      if (yr) {
        const float4 u = ld4(yr + w);
        v.x += u.x, v.y += u.y, v.z += u.z, v.w += u.w;
        st4(xr + w, v);
      }
      st4(row + w, v);
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
  } else {
    for (int64_t w = threadIdx.x; w < W; w += blockDim.x) {
      float v = xr[w];
      if (yr) {
        v += yr[w];
        xr[w] = v;
      }
      row[w] = v;
      ss = fmaf(v, v, ss);
    }
  }
  if (!weight) return;
  const float k = 1.f / sqrtf(block_sum(ss, scratch) / (float)W + eps);
  if (VEC) {
    for (int64_t w = (int64_t)threadIdx.x * 4; w < W; w += (int64_t)blockDim.x * 4) {
      const float4 v = ld4(row + w), g = ld4(weight + w);
      st4(out + i * W + w, make_float4(v.x * k * g.x, v.y * k * g.y, v.z * k * g.z, v.w * k * g.w));
    }
  } else {
    for (int64_t w = threadIdx.x; w < W; w += blockDim.x) stf(out + i * W + w, row[w] * k * ldf(weight + w));
  }
}

// pos * z^2 + z / 2 above zero, neg * (exp(z) - 1 - z) + z / 2 below it
__device__ __forceinline__ float xielu(float z, float pos, float neg) {
  const float r = z > 0.f ? pos * z * z : neg * (expm1f(z) - z);
  return fmaf(0.5f, z, r);
}

template <typename T, bool VEC>
__global__ void xielu_rows_kernel(const float* __restrict__ in, int64_t ld, int64_t cols, float pos, float neg, T* __restrict__ out,
                                  int64_t ld_out) {
  const float* src = in + (int64_t)blockIdx.x * ld;
  T* dst = out + (int64_t)blockIdx.x * ld_out;
  const int64_t i0 = (int64_t)blockIdx.y * blockDim.x + threadIdx.x, step = (int64_t)gridDim.y * blockDim.x;
  if (VEC) {
    for (int64_t c = i0 * 4; c < cols; c += step * 4) {
      const float4 z = ld4(src + c);
      st4(dst + c, make_float4(xielu(z.x, pos, neg), xielu(z.y, pos, neg), xielu(z.z, pos, neg), xielu(z.w, pos, neg)));
    }
  } else {
    for (int64_t c = i0; c < cols; c += step) stf(dst + c, xielu(src[c], pos, neg));
  }
}

inline bool on(const void* p, size_t bytes) { return reinterpret_cast<uintptr_t>(p) % bytes == 0; }

}  // namespace

extern "C" int ao_lm_embed_scaled(const void* table, int dt, const int64_t* tok, int64_t n, int64_t width, float scale, float* x,
                                  void* stream) {
  LM_CHECK_ARG(table && tok && x && n > 0 && width > 0);
  LM_DISPATCH(dt, embed_scaled_kernel<T><<<(unsigned)n, width >= 1024 ? 256 : 128, 0, lm_stream(stream)>>>(
                      static_cast<const T*>(table), tok, width, scale, x));
  return lm_launch_status();
}

extern "C" int ao_lm_add_rms_norm(float* x, const float* y, const int32_t* rows, int64_t m, int64_t width, const void* weight, int dt,
                                  float eps, void* out, void* stream) {
  LM_CHECK_ARG(x && m > 0 && width > 0 && (weight || y) && (!weight || out) && !(y && rows));
  const size_t smem = (size_t)width * sizeof(float);
  if (smem > 200 * 1024) return AO_B200_ERR_UNSUPPORTED;
  // four values per thread: a row of a few thousand values is one access deep
  const int64_t want = ((width / 4 + 31) / 32) * 32, cap = m < 296 ? 1024 : 512;
  const unsigned th = (unsigned)(want < 64 ? 64 : want > cap ? cap : want);
  LM_DISPATCH(dt, {
    const bool vec = width % 4 == 0 && on(x, 16) && on(y, 16) && on(weight, 4 * sizeof(T)) && on(out, 4 * sizeof(T));
    auto kern = vec ? add_rms_norm_kernel<T, true> : add_rms_norm_kernel<T, false>;
    if (smem > 40 * 1024) {
      static bool set[2] = {false, false};
      if (!set[vec]) {
        if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return AO_B200_ERR_CUDA;
        set[vec] = true;
      }
    }
    kern<<<(unsigned)m, th, smem, lm_stream(stream)>>>(x, y, rows, width, static_cast<const T*>(weight), eps, static_cast<T*>(out));
  });
  return lm_launch_status();
}

extern "C" int ao_lm_xielu_rows(const float* in, int64_t ld, int64_t n, int64_t cols, float pos, float neg, void* out, int64_t ld_out,
                                int dt, void* stream) {
  LM_CHECK_ARG(in && out && n > 0 && cols > 0 && ld >= cols && ld_out >= cols);
  LM_DISPATCH(dt, {
    const bool vec = cols % 4 == 0 && ld % 4 == 0 && ld_out % 4 == 0 && on(in, 16) && on(out, 4 * sizeof(T));
    const int64_t items = vec ? cols / 4 : cols;
    int64_t parts = (items + 511) / 512;      // two or so accesses per thread
    if (parts > 64) parts = 64;
    const dim3 grid((unsigned)n, (unsigned)parts);
    if (vec)
      xielu_rows_kernel<T, true><<<grid, 256, 0, lm_stream(stream)>>>(in, ld, cols, pos, neg, static_cast<T*>(out), ld_out);
    else
      xielu_rows_kernel<T, false><<<grid, 256, 0, lm_stream(stream)>>>(in, ld, cols, pos, neg, static_cast<T*>(out), ld_out);
  });
  return lm_launch_status();
}

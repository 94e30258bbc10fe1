// Row kernels of designs that norm a sublayer's input AND its result with layer norms (a weight, no bias) around an fp32
// residual, and of spans of layers that are run several times with the embedding output fed in again in front of every pass:
//     ao_lm_post_layer_norm_residual   residual += norm(result), the next sublayer's norm (or the residual in the storage type,
//                                      the operand of a pass's input product) while the row is in registers; or residual =
//                                      sum of two products, with the first norm of a pass
//     ao_lm_embed_bigram               scaled embedding + a row of a hashed table of (previous token, token) pairs; the slot's
//                                      last token is the state
#include "lm_common.cuh"

using namespace lm;

namespace {

constexpr int kMaxWarps = 32;

// Sum over the block; every thread gets it.  scratch: kMaxWarps floats that no other sum of the kernel uses (one barrier per sum).
__device__ __forceinline__ float block_total(float v, float* scratch) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = blockDim.x >> 5;
  v = warp_sum(v);
  if (nw == 1) return v;
  if (lane == 0) scratch[w] = v;
  __syncthreads();
  return warp_sum(lane < nw ? scratch[lane] : 0.f);
}

// A thread's share of a row: PER groups of four values.  VEC: group j is the four neighbours at 4 (threadIdx + j blockDim);
// otherwise value 4 j + e is at threadIdx + (4 j + e) blockDim.
template <int PER, bool VEC>
struct RowShare {
  static __device__ __forceinline__ int64_t at(int j, int e) {
    return VEC ? ((int64_t)threadIdx.x + (int64_t)j * blockDim.x) * 4 + e : (int64_t)threadIdx.x + (int64_t)(4 * j + e) * blockDim.x;
  }
  template <typename U>
  static __device__ __forceinline__ void load(const U* __restrict__ p, int64_t W, float (&v)[PER * 4]) {
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      if (VEC) {
        const int64_t w = at(j, 0);
        const float4 u = w < W ? ld4(p + w) : make_float4(0.f, 0.f, 0.f, 0.f);
        v[4 * j] = u.x, v[4 * j + 1] = u.y, v[4 * j + 2] = u.z, v[4 * j + 3] = u.w;
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) v[4 * j + e] = at(j, e) < W ? ldf(p + at(j, e)) : 0.f;
      }
    }
  }
  template <typename U>
  static __device__ __forceinline__ void store(U* __restrict__ p, int64_t W, const float (&v)[PER * 4]) {
#pragma unroll
    for (int j = 0; j < PER; ++j) {
      if (VEC) {
        const int64_t w = at(j, 0);
        if (w < W) st4(p + w, make_float4(v[4 * j], v[4 * j + 1], v[4 * j + 2], v[4 * j + 3]));
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (at(j, e) < W) stf(p + at(j, e), v[4 * j + e]);
      }
    }
  }
  // v = (v - mean) / sqrt(mean squared deviation + eps) * g; scratch: two sums' worth
  static __device__ __forceinline__ void norm(int64_t W, float eps, const float (&g)[PER * 4], float (&v)[PER * 4], float (*scratch)[kMaxWarps]) {
    float s = 0.f, ss = 0.f;
#pragma unroll
    for (int i = 0; i < PER * 4; ++i) s += v[i];             // places past the row hold zeros
    const float mean = block_total(s, scratch[0]) / (float)W;
#pragma unroll
    for (int i = 0; i < PER * 4; ++i) {
      v[i] = at(i / 4, i % 4) < W ? v[i] - mean : 0.f;
      ss = fmaf(v[i], v[i], ss);
    }
    const float k = 1.f / sqrtf(block_total(ss, scratch[1]) / (float)W + eps);
#pragma unroll
    for (int i = 0; i < PER * 4; ++i) v[i] *= k * g[i];
  }
};

struct PostArgs {
  float* x;
  const float *y, *y_bias, *add_rows;
  const void *post_w, *next_w;
  int64_t W, ld_y, ld_add, ld_out;
  float eps;
  int replace;
  void* out;
};

template <typename T, int PER, bool VEC>
__global__ void __launch_bounds__(1024) post_layer_norm_kernel(PostArgs a) {
  using Share = RowShare<PER, VEC>;
  __shared__ float scratch[4][kMaxWarps];
  const int64_t t = blockIdx.x, W = a.W;
  const T *post_w = static_cast<const T*>(a.post_w), *next_w = static_cast<const T*>(a.next_w);
  float* xr = a.x + t * W;
  float x[PER * 4], v[PER * 4], u[PER * 4];
  pdl_trigger();
  pdl_wait();
  // every load of the row is in flight before the first reduction
  if (!a.replace) {
    Share::load(xr, W, x);
  } else {
#pragma unroll
    for (int i = 0; i < PER * 4; ++i) x[i] = 0.f;
  }
  if (a.y) {
    Share::load(a.y + t * a.ld_y, W, v);
    if (a.y_bias) {
      Share::load(a.y_bias, W, u);
#pragma unroll
      for (int i = 0; i < PER * 4; ++i) v[i] += u[i];
    }
    if (post_w) {
      Share::load(post_w, W, u);
      Share::norm(W, a.eps, u, v, scratch);
    }
#pragma unroll
    for (int i = 0; i < PER * 4; ++i) x[i] += v[i];
    if (a.add_rows) {
      Share::load(a.add_rows + t * a.ld_add, W, v);
#pragma unroll
      for (int i = 0; i < PER * 4; ++i) x[i] += v[i];
    }
    Share::store(xr, W, x);
  }
  if (!a.out) return;
  T* out = static_cast<T*>(a.out) + t * a.ld_out;
  if (next_w) {
    Share::load(next_w, W, u);
    Share::norm(W, a.eps, u, x, scratch + 2);
  }
  Share::store(out, W, x);
}

template <typename T, bool VEC>
__global__ void embed_bigram_kernel(const T* __restrict__ table, const T* __restrict__ bigram, const int64_t* __restrict__ tok, int64_t W,
                                    float scale, int64_t buckets, int64_t mul_prev, int64_t mul_cur, int64_t* __restrict__ last,
                                    const int32_t* __restrict__ slot, const int32_t* __restrict__ pos, const int32_t* __restrict__ back,
                                    const int32_t* __restrict__ ahead, float* __restrict__ x, T* __restrict__ out) {
  __shared__ int64_t shared_row;
  pdl_trigger();
  pdl_wait();
  const int64_t t = blockIdx.x, token = tok[t];
  if (bigram) {
    if (threadIdx.x == 0) {
      int64_t prev = -1;
      if (back[t] > 0) {
        prev = tok[t - 1];
      } else {
        // the segment's first row reads the slot's last token and puts the segment's last token in its place: reader and
        // writer are one thread, whatever order the rows run in
        int64_t* mem = last + slot[t];
        if (pos[t] > 0) prev = *mem;
        *mem = tok[t + ahead[t]];
      }
      int64_t r = buckets;
      if (prev >= 0) {
        r = (prev * mul_prev + token * mul_cur) % buckets;
        if (r < 0) r += buckets;
      }
      shared_row = r;
    }
    __syncthreads();
  }
  const T* e = table + token * W;
  const T* b = bigram ? bigram + shared_row * W : nullptr;
  if (VEC) {
    for (int64_t w = (int64_t)threadIdx.x * 4; w < W; w += (int64_t)blockDim.x * 4) {
      const float4 p = ld4(e + w), q = b ? ld4(b + w) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 v = make_float4(fmaf(p.x, scale, q.x), fmaf(p.y, scale, q.y), fmaf(p.z, scale, q.z), fmaf(p.w, scale, q.w));
      st4(x + t * W + w, v);
      if (out) st4(out + t * W + w, v);
    }
  } else {
    for (int64_t w = threadIdx.x; w < W; w += blockDim.x) {
      const float v = fmaf(ldf(e + w), scale, b ? ldf(b + w) : 0.f);
      x[t * W + w] = v;
      if (out) stf(out + t * W + w, v);
    }
  }
}

inline bool on(const void* p, size_t bytes) { return reinterpret_cast<uintptr_t>(p) % bytes == 0; }

template <typename T, bool VEC>
int launch_post(const PostArgs& a, int64_t n, cudaStream_t st) {
  // groups of four values per thread: many rows fill the GPU with small blocks, few rows want each row spread over a large one
  const int64_t groups = (a.W + 3) / 4, spread = n < 296 ? 1 : groups <= 128 ? 1 : 2;
  int64_t th = ((groups + spread - 1) / spread + 31) / 32 * 32;
  th = th < 32 ? 32 : th > 1024 ? 1024 : th;
  const int64_t per = (groups + th - 1) / th;
  const dim3 grid((unsigned)n), block((unsigned)th);
  if (per <= 1) return lm_launch_early(post_layer_norm_kernel<T, 1, VEC>, grid, block, 0, st, a);
  if (per <= 2) return lm_launch_early(post_layer_norm_kernel<T, 2, VEC>, grid, block, 0, st, a);
  if (per <= 4) return lm_launch_early(post_layer_norm_kernel<T, 4, VEC>, grid, block, 0, st, a);
  if (per <= 8) return lm_launch_early(post_layer_norm_kernel<T, 8, VEC>, grid, block, 0, st, a);
  return AO_B200_ERR_UNSUPPORTED;
}

}  // namespace

extern "C" int ao_lm_post_layer_norm_residual(float* x, const float* y, int64_t ld_y, const float* y_bias, const void* post_w,
                                              const float* add_rows, int64_t ld_add, int replace, const void* next_w, int dt, float eps,
                                              int64_t n, int64_t width, void* out, int64_t ld_out, void* stream) {
  LM_CHECK_ARG(x && n > 0 && width > 0 && (y || (!y_bias && !post_w && !add_rows && !replace)) && (y || out) && (out || !next_w));
  LM_CHECK_ARG((!y || ld_y >= width) && (!add_rows || ld_add >= width) && (!out || ld_out >= width));
  const PostArgs a{x, y, y_bias, add_rows, post_w, next_w, width, ld_y, ld_add, ld_out, eps, replace, out};
  LM_DISPATCH(dt, {
    const bool vec = width % 4 == 0 && (!y || ld_y % 4 == 0) && (!add_rows || ld_add % 4 == 0) && (!out || ld_out % 4 == 0) && on(x, 16) &&
                     on(y, 16) && on(y_bias, 16) && on(add_rows, 16) && on(post_w, 4 * sizeof(T)) && on(next_w, 4 * sizeof(T)) &&
                     on(out, 4 * sizeof(T));
    return vec ? launch_post<T, true>(a, n, lm_stream(stream)) : launch_post<T, false>(a, n, lm_stream(stream));
  });
  return AO_B200_OK;
}

extern "C" int ao_lm_embed_bigram(const void* table, const void* bigram, int dt, const int64_t* tok, int64_t n, int64_t width, float scale,
                                  int64_t buckets, int64_t mul_prev, int64_t mul_cur, int64_t* last, const int32_t* slot,
                                  const int32_t* pos, const int32_t* back, const int32_t* ahead, float* x, void* out, void* stream) {
  LM_CHECK_ARG(table && tok && x && n > 0 && width > 0);
  LM_CHECK_ARG(!bigram || (buckets > 0 && last && slot && pos && back && ahead));
  const int64_t want = ((width + 3) / 4 + 31) / 32 * 32, cap = n < 296 ? 1024 : 256;
  const unsigned th = (unsigned)(want > cap ? cap : want);
  LM_DISPATCH(dt, {
    const bool vec = width % 4 == 0 && on(table, 4 * sizeof(T)) && on(bigram, 4 * sizeof(T)) && on(x, 16) && on(out, 4 * sizeof(T));
    auto kern = vec ? embed_bigram_kernel<T, true> : embed_bigram_kernel<T, false>;
    return lm_launch_early(kern, dim3((unsigned)n), dim3(th), 0, lm_stream(stream), static_cast<const T*>(table), static_cast<const T*>(bigram),
                           tok, width, scale, buckets, mul_prev, mul_cur, last, slot, pos, back, ahead, x, static_cast<T*>(out));
  });
  return AO_B200_OK;
}

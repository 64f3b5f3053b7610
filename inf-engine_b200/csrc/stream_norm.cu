// The sum of one or several sublayers' results into the float32 residual stream, with a multiplier, and the norm that the
// stream meets next, in one kernel:
//
//   x = residual[row] + mult * scale * (y[row] + sum_e extra_e[row])
//                                                             (scale [d] optional: 1; y optional: nothing is added)
//   y[row] = sum_r weight[row, r] * y_pairs[row * top + r]     (a mixture of experts hands over its choices' results
//                                                               and their weights; r upward)
//   extra_0, extra_1                                          (what other sublayers that read the same input return)
//   residual[row] = x                                         (unless rows are gathered)
//   out[m] = x / rms * gain,   rms of each of `groups` equal consecutive parts of the row by itself:
//            sqrt(mean(part^2) + eps)
//   or      tanh(alpha x) * gain + bias, coordinate by coordinate
//
// `out` may be left out (the sum alone).
//
// The root mean square: one block per row.  The new row is staged in shared memory; the sum of squares of a part is formed
// by one warp or by several that take equal pieces of it, whose sums are then added in order: a row's result depends on
// the row alone.  The hyperbolic tangent needs nothing of the rest of the row: a thread per coordinate (or four), spread
// over as many blocks as that makes.  The row moves in pieces of four elements where sizes and strides allow it.
#include "common.cuh"

#define SN_THREADS 256
#define SN_WARPS (SN_THREADS / 32)
#define SN_EXTRAS 2

struct StreamNormParams {
  float* residual;
  const void* y;
  const float* scale;
  const float* weights;   // [rows, top] or null
  const void* gain;
  void* out;
  const int* row_index;
  int y_stride, top, d, groups, pieces;
  float eps;
  float mult;
  const void* extra[SN_EXTRAS];   // rows of the activation type, or null
  int extra_stride[SN_EXTRAS];
  int extra_f32;
  const void* bias;               // the tanh form
  float alpha;
};

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<bf16>(const bf16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<const unsigned*>(&a);
  raw.y = *reinterpret_cast<const unsigned*>(&b);
  *reinterpret_cast<uint2*>(p) = raw;
}

// the multiplied summand of coordinates i .. i + 3 (or of coordinate i) of a row
template <typename TY>
__device__ __forceinline__ float4 summand4(const StreamNormParams& p, const TY* y, const float* wt, int row, int i) {
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
  if (wt == nullptr) {
    a = load4<TY>(y + i);
  } else {
    for (int r = 0; r < p.top; ++r) {
      const float4 v = load4<TY>(y + (size_t)r * p.y_stride + i);
      const float w = wt[r];
      a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
    }
  }
#pragma unroll
  for (int e = 0; e < SN_EXTRAS; ++e) {
    if (p.extra[e] == nullptr) continue;
    const size_t at = (size_t)row * p.extra_stride[e] + i;
    const float4 v = p.extra_f32 ? load4<float>((const float*)p.extra[e] + at) : load4<bf16>((const bf16*)p.extra[e] + at);
    a.x += v.x; a.y += v.y; a.z += v.z; a.w += v.w;
  }
  float4 s = p.scale ? load4<float>(p.scale + i) : make_float4(1.f, 1.f, 1.f, 1.f);
  if (p.mult != 1.f) { s.x *= p.mult; s.y *= p.mult; s.z *= p.mult; s.w *= p.mult; }
  return make_float4(s.x * a.x, s.y * a.y, s.z * a.z, s.w * a.w);
}
template <typename TY>
__device__ __forceinline__ float summand1(const StreamNormParams& p, const TY* y, const float* wt, int row, int i) {
  float a = 0.f;
  if (wt == nullptr) a = to_f32(y[i]);
  else
    for (int r = 0; r < p.top; ++r) a = fmaf(wt[r], to_f32(y[(size_t)r * p.y_stride + i]), a);
#pragma unroll
  for (int e = 0; e < SN_EXTRAS; ++e) {
    if (p.extra[e] == nullptr) continue;
    const size_t at = (size_t)row * p.extra_stride[e] + i;
    a += p.extra_f32 ? ((const float*)p.extra[e])[at] : to_f32(((const bf16*)p.extra[e])[at]);
  }
  return (p.scale ? p.scale[i] : 1.f) * p.mult * a;
}

template <typename TY, typename TW, typename TA, int VEC>
__global__ void __launch_bounds__(SN_THREADS) stream_norm_kernel(StreamNormParams p) {
  extern __shared__ __align__(16) float xs[];
  __shared__ float part_sum[SN_WARPS];
  float* inv = xs + ((p.d + 3) & ~3);          // [groups]
  pdl_trigger();
  pdl_wait();
  const int m = blockIdx.x;
  const int row = p.row_index ? p.row_index[m] : m;
  float* res = p.residual + (size_t)row * p.d;
  const TY* y = p.y ? (const TY*)p.y + (size_t)row * p.top * p.y_stride : nullptr;
  const float* wt = p.weights ? p.weights + (size_t)row * p.top : nullptr;
  const bool keep = y != nullptr && p.row_index == nullptr;
  for (int i = threadIdx.x * VEC; i < p.d; i += SN_THREADS * VEC) {
    if constexpr (VEC == 4) {
      float4 x = load4<float>(res + i);
      if (y != nullptr) {
        const float4 a = summand4<TY>(p, y, wt, row, i);
        x.x += a.x; x.y += a.y; x.z += a.z; x.w += a.w;
        if (keep) store4(res + i, x);
      }
      store4(xs + i, x);
    } else {
      float x = res[i];
      if (y != nullptr) {
        x += summand1<TY>(p, y, wt, row, i);
        if (keep) res[i] = x;
      }
      xs[i] = x;
    }
  }
  if (p.out == nullptr) return;
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int size = p.d / p.groups;
  // `pieces` warps a part (a power of two up to the block's warps): each sums its piece, one thread adds them in order
  for (int g0 = 0; g0 < p.groups; g0 += SN_WARPS / p.pieces) {
    const int g = g0 + warp / p.pieces, piece = warp % p.pieces;
    float ss = 0.f;
    if (g < p.groups) {
      const int len = (size + p.pieces - 1) / p.pieces;
      const int lo = piece * len, hi = min(size, lo + len);
      const float* part = xs + (size_t)g * size;
      for (int i = lo + lane; i < hi; i += 32) ss = fmaf(part[i], part[i], ss);
    }
    ss = warp_sum(ss);
    if (p.pieces == 1) {
      if (lane == 0 && g < p.groups) inv[g] = sqrtf(ss / (float)size + p.eps);
    } else {
      if (lane == 0) part_sum[warp] = ss;
      __syncthreads();
      if (lane == 0 && piece == 0 && g < p.groups) {
        float total = 0.f;
        for (int k = 0; k < p.pieces; ++k) total += part_sum[warp + k];
        inv[g] = sqrtf(total / (float)size + p.eps);
      }
      __syncthreads();
    }
  }
  __syncthreads();
  TA* o = (TA*)p.out + (size_t)m * p.d;
  const TW* gain = (const TW*)p.gain;
  for (int i = threadIdx.x * VEC; i < p.d; i += SN_THREADS * VEC) {
    if constexpr (VEC == 4) {
      // (a part's size is a multiple of four: the four share its root mean square)
      const float r = inv[i / size];
      const float4 x = load4<float>(xs + i), w = load4<TW>(gain + i);
      store4(o + i, make_float4(x.x / r * w.x, x.y / r * w.y, x.z / r * w.z, x.w / r * w.w));
    } else {
      o[i] = from_f32<TA>(xs[i] / inv[i / size] * to_f32(gain[i]));
    }
  }
}

// The tanh form: block (x, m) takes SN_THREADS pieces of row m.
template <typename TY, typename TW, typename TA, int VEC>
__global__ void __launch_bounds__(SN_THREADS) stream_tanh_kernel(StreamNormParams p) {
  pdl_trigger();
  const int i = (blockIdx.x * SN_THREADS + threadIdx.x) * VEC;
  if (i >= p.d) return;
  const TW* gain = (const TW*)p.gain + i;
  const TW* bias = (const TW*)p.bias + i;
  const int m = blockIdx.y;
  if constexpr (VEC == 4) {
    const float4 w = load4<TW>(gain), b = load4<TW>(bias);      // constant data: fetched before the kernel ahead has finished
    pdl_wait();
    const int row = p.row_index ? p.row_index[m] : m;
    float* res = p.residual + (size_t)row * p.d + i;
    float4 x = load4<float>(res);
    if (p.y != nullptr) {
      const float4 a = summand4<TY>(p, (const TY*)p.y + (size_t)row * p.top * p.y_stride,
                                    p.weights ? p.weights + (size_t)row * p.top : nullptr, row, i);
      x.x += a.x; x.y += a.y; x.z += a.z; x.w += a.w;
      if (p.row_index == nullptr) store4(res, x);
    }
    store4((TA*)p.out + (size_t)m * p.d + i,
           make_float4(fmaf(tanhf(p.alpha * x.x), w.x, b.x), fmaf(tanhf(p.alpha * x.y), w.y, b.y),
                       fmaf(tanhf(p.alpha * x.z), w.z, b.z), fmaf(tanhf(p.alpha * x.w), w.w, b.w)));
  } else {
    pdl_wait();
    const int row = p.row_index ? p.row_index[m] : m;
    float* res = p.residual + (size_t)row * p.d + i;
    float x = *res;
    if (p.y != nullptr) {
      x += summand1<TY>(p, (const TY*)p.y + (size_t)row * p.top * p.y_stride,
                        p.weights ? p.weights + (size_t)row * p.top : nullptr, row, i);
      if (p.row_index == nullptr) *res = x;
    }
    ((TA*)p.out)[(size_t)m * p.d + i] = from_f32<TA>(fmaf(tanhf(p.alpha * x), to_f32(*gain), to_f32(*bias)));
  }
}

template <typename TY, typename TW, typename TA>
static int launch_stream_norm(const StreamNormParams& p, int n_rows, cudaStream_t stream) {
  if (p.bias != nullptr) {
    uintptr_t at = (uintptr_t)p.residual | (uintptr_t)p.y | (uintptr_t)p.scale | (uintptr_t)p.gain | (uintptr_t)p.out |
                   (uintptr_t)p.bias;
    bool vec = (p.d % 4) == 0 && (p.y_stride % 4) == 0;
    for (int e = 0; e < SN_EXTRAS; ++e) { at |= (uintptr_t)p.extra[e]; vec = vec && (p.extra_stride[e] % 4) == 0; }
    vec = vec && (at & 15) == 0;
    if (n_rows > 65535) return IE_BAD_SIZE;
    const int per = SN_THREADS * (vec ? 4 : 1);
    dim3 grid((p.d + per - 1) / per, n_rows);
    if (vec) return launch_k(stream_tanh_kernel<TY, TW, TA, 4>, grid, SN_THREADS, 0, stream, p);
    return launch_k(stream_tanh_kernel<TY, TW, TA, 1>, grid, SN_THREADS, 0, stream, p);
  }
  const size_t smem = sizeof(float) * (((size_t)p.d + 3) / 4 * 4 + p.groups);
  if (smem > 200 * 1024) return IE_BAD_SIZE;
  uintptr_t at = (uintptr_t)p.residual | (uintptr_t)p.y | (uintptr_t)p.scale | (uintptr_t)p.gain | (uintptr_t)p.out;
  bool vec = (p.d % 4) == 0 && (p.d / p.groups) % 4 == 0 && (p.y_stride % 4) == 0;
  for (int e = 0; e < SN_EXTRAS; ++e) { at |= (uintptr_t)p.extra[e]; vec = vec && (p.extra_stride[e] % 4) == 0; }
  vec = vec && (at & 15) == 0;
  auto kernel = vec ? stream_norm_kernel<TY, TW, TA, 4> : stream_norm_kernel<TY, TW, TA, 1>;
  if (smem > 47 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return launch_k(kernel, n_rows, SN_THREADS, smem, stream, p);
}

// bias == null: the root mean square (gain, groups, eps); else tanh(alpha x) * gain + bias (bias of the gain's type).
// extra_0, extra_1: rows of one type, or null (without y there are none).
extern "C" int ie_stream_norm(float* residual, const void* y, int y_dtype, int y_stride, const float* scale, float mult,
                              const float* weights, int top, const void* extra_0, int extra_0_stride, const void* extra_1,
                              int extra_1_stride, int extra_dtype, const void* gain, int gain_dtype, int groups, float eps,
                              const void* bias, float alpha, void* out, int out_dtype, const int* row_index, int n_rows,
                              int d, cudaStream_t stream) {
  if (n_rows <= 0) return IE_OK;
  if (d <= 0 || groups <= 0 || d % groups || top <= 0 || (top > 1 && weights == nullptr)) return IE_BAD_SIZE;
  if (out != nullptr && gain == nullptr) return IE_BAD_SIZE;
  if (bias != nullptr && out == nullptr) return IE_BAD_SIZE;
  if (y == nullptr && (extra_0 != nullptr || extra_1 != nullptr)) return IE_BAD_SIZE;
  if (extra_dtype != IE_F32 && extra_dtype != IE_BF16) return IE_BAD_DTYPE;
  StreamNormParams p;
  p.residual = residual; p.y = y; p.scale = scale; p.weights = weights; p.gain = gain; p.out = out;
  p.row_index = row_index; p.y_stride = y != nullptr ? y_stride : d; p.top = top; p.d = d; p.groups = groups; p.eps = eps;
  p.pieces = groups > 4 ? 1 : (groups > 2 ? 2 : (groups == 2 ? 4 : 8));      // SN_WARPS / pieces parts at a time
  p.mult = mult; p.bias = bias; p.alpha = alpha; p.extra_f32 = extra_dtype == IE_F32;
  p.extra[0] = extra_0; p.extra[1] = extra_1;
  p.extra_stride[0] = extra_0 != nullptr ? extra_0_stride : 0;
  p.extra_stride[1] = extra_1 != nullptr ? extra_1_stride : 0;
  if (y == nullptr) y_dtype = IE_F32;
  if (out == nullptr) { out_dtype = IE_F32; gain_dtype = IE_F32; }
#define SN_OUT(TY, TW)                                                                       \
  {                                                                                          \
    if (out_dtype == IE_F32) return launch_stream_norm<TY, TW, float>(p, n_rows, stream);    \
    if (out_dtype == IE_BF16) return launch_stream_norm<TY, TW, bf16>(p, n_rows, stream);    \
  }
  if (y_dtype == IE_F32 && gain_dtype == IE_F32) SN_OUT(float, float);
  if (y_dtype == IE_F32 && gain_dtype == IE_BF16) SN_OUT(float, bf16);
  if (y_dtype == IE_BF16 && gain_dtype == IE_F32) SN_OUT(bf16, float);
  if (y_dtype == IE_BF16 && gain_dtype == IE_BF16) SN_OUT(bf16, bf16);
#undef SN_OUT
  return IE_BAD_DTYPE;
}

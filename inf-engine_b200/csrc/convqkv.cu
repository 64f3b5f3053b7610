// From the raw projections of a token's queries, keys and values to what attention reads, in one kernel:
//   * a short causal convolution over time, a filter per channel:  y_t = sum_j w[j, c] u_(t - (taps - 1) + j), where the
//     u before the step's first token come from the request's state ([taps - 1, channels], oldest first, zeros when the
//     sequence starts), which is then moved on by the step's tokens;
//   * a rotation by position of the first `rot_dims` dimensions of every query and key head, in neighbouring pairs or in
//     halves: (u, v) -> (u cos a - v sin a, v cos a + u sin a) * mult, a = position * inv_freq[i] (float64 frequencies,
//     the angle brought into one turn in double, sine and cosine float32);
//   * values kept for later layers of the step (v_mode 1), or blended with the values an earlier layer kept:
//     v <- (1 - lambda) v + lambda v_kept (v_mode 2);
//   * queries to `q_out`, keys and values to the tokens' page slots.
// Sums, angles and the blend are float32.  A row of `x` holds queries, keys and values at the columns k0 and v0 (a
// multiple of 8 each; columns between them belong to nobody), heads side by side.  Filters and state are laid out over
// the same columns.  A token's output is the same however the sequence was cut into steps.
//
// Two forms.  `conv_qkv_kernel`: any sizes and types; a block takes a head of one request and a chunk of tokens, a
// thread a dimension (and, for a rotated one, its partner's convolution too).  `conv_qkv_vec_kernel`: bfloat16, head
// sizes that are multiples of 8, neighbouring pairs, up to 8 taps; a thread takes 8 channels (16 bytes) and walks the
// tokens of a chunk with the last inputs in registers, so a row is read once; the chunk's sines and cosines are worked
// out once a block and shared by all heads.  In both, only a request's first chunk reads the old state, and the block
// (the thread) that read it writes the new one.
#include "common.cuh"

#define CQ_MAX_TAPS 16
#define CQ_VEC_TAPS 8

struct ConvQkvParams {
  const void* x;
  int x_stride;
  const float* w;          // [taps, channels] (null: no convolution, taps is 1)
  void* state;             // slots of [taps - 1, channels]
  long long state_stride;  // elements between two slots
  int channels, taps;
  void* q_out;
  int q_stride;
  void* kpool;
  void* vpool;
  void* v_kept;            // [tokens, kv heads * hd_v]
  int v_mode;
  float lambda;
  const double* inv_freq;
  int rot_dims, neighbours;
  float mult;
  const int* positions;
  const int* slot_mapping;
  const int* q_start;
  const int* slots;
  int heads, kv_heads, hd, hd_v, k0, v0, page_size, write_state;
};

__device__ __forceinline__ void turn(double position, double freq, float mult, float& cs, float& sn) {
  const double turns = position * freq * 0.15915494309189535;
  sincosf((float)((turns - floor(turns)) * 6.283185307179586), &sn, &cs);
  cs *= mult;
  sn *= mult;
}

#define CQ_TL 4
#define CQ_CHUNK 32

template <typename T>
__device__ __forceinline__ float conv_at(const ConvQkvParams& p, const T* __restrict__ st, int q0, int t, int c) {
  const T* x = (const T*)p.x;
  if (p.w == nullptr) return to_f32(x[(size_t)t * p.x_stride + c]);
  float acc = 0.f;
  for (int j = 0; j < p.taps; ++j) {
    const int src = t - (p.taps - 1) + j;
    float u = 0.f;
    if (src >= q0) u = to_f32(x[(size_t)src * p.x_stride + c]);
    else if (st != nullptr) u = to_f32(st[(size_t)(p.taps - 1 - (q0 - src)) * p.channels + c]);
    acc = fmaf(p.w[(size_t)j * p.channels + c], u, acc);
  }
  return acc;
}

template <typename T>
__global__ void __launch_bounds__(32 * CQ_TL) conv_qkv_kernel(ConvQkvParams p) {
  pdl_trigger();
  pdl_wait();
  const int req = blockIdx.y;
  const int q0 = p.q_start[req], q1 = p.q_start[req + 1];
  const int t_lo = q0 + blockIdx.z * CQ_CHUNK, t_hi = min(q1, t_lo + CQ_CHUNK);
  if (t_lo >= q1) return;
  const int item = blockIdx.x;                          // a query head, a key head or a value head
  const int side = item < p.heads ? 0 : (item < p.heads + p.kv_heads ? 1 : 2);
  const int h = side == 0 ? item : (side == 1 ? item - p.heads : item - p.heads - p.kv_heads);
  const int hd = side == 2 ? p.hd_v : p.hd;
  const int c0 = (side == 0 ? 0 : (side == 1 ? p.k0 : p.v0)) + h * hd;
  const int slot = p.slots != nullptr ? IE_SLOT(p.slots[req]) : -1;
  T* st = (slot >= 0 && p.state != nullptr && p.taps > 1) ? (T*)p.state + (size_t)slot * p.state_stride : nullptr;
  const int half = p.rot_dims >> 1;
  for (int t = t_lo + threadIdx.y; t < t_hi; t += CQ_TL) {
    const int page_slot = p.slot_mapping != nullptr ? IE_SLOT(p.slot_mapping[t]) : -1;
    const int page = page_slot >= 0 ? page_slot / p.page_size : 0, off = page_slot >= 0 ? page_slot % p.page_size : 0;
    for (int d = threadIdx.x; d < hd; d += 32) {
      float y = conv_at<T>(p, st, q0, t, c0 + d);
      if (side != 2 && p.inv_freq != nullptr && d < p.rot_dims) {
        int pair, partner;
        bool first;
        if (p.neighbours) {
          pair = d >> 1; first = !(d & 1); partner = d ^ 1;
        } else {
          first = d < half; pair = first ? d : d - half; partner = first ? d + half : d - half;
        }
        const float z = conv_at<T>(p, st, q0, t, c0 + partner);
        float cs, sn;
        turn((double)p.positions[t], p.inv_freq[pair], p.mult, cs, sn);
        y = first ? fmaf(y, cs, -z * sn) : fmaf(y, cs, z * sn);
      }
      if (side == 0) {
        ((T*)p.q_out)[(size_t)t * p.q_stride + h * hd + d] = from_f32<T>(y);
        continue;
      }
      if (side == 1) {
        if (page_slot >= 0 && p.kpool != nullptr)
          ((T*)p.kpool)[(((size_t)page * p.kv_heads + h) * p.page_size + off) * hd + d] = from_f32<T>(y);
        continue;
      }
      T* kept = p.v_mode ? (T*)p.v_kept + (size_t)t * p.kv_heads * hd + h * hd + d : nullptr;
      if (p.v_mode == 1) *kept = from_f32<T>(y);
      if (p.v_mode == 2) y = fmaf(p.lambda, to_f32(*kept), (1.f - p.lambda) * y);
      if (page_slot >= 0 && p.vpool != nullptr)
        ((T*)p.vpool)[(((size_t)page * p.kv_heads + h) * p.page_size + off) * hd + d] = from_f32<T>(y);
    }
  }
  if (blockIdx.z > 0 || st == nullptr || !p.write_state) return;
  __syncthreads();                                       // every row of threads has read what it needs of the old state
  if (threadIdx.y != 0) return;
  const T* x = (const T*)p.x;
  const int n = q1 - q0, keep = p.taps - 1;
  for (int d = threadIdx.x; d < hd; d += 32) {
    const int c = c0 + d;
    // place i takes the input of token q1 - keep + i, or what stood n places further on; ascending i reads ahead of its writes
    for (int i = 0; i < keep; ++i) {
      const int src = q1 - keep + i;
      st[(size_t)i * p.channels + c] = src >= q0 ? x[(size_t)src * p.x_stride + c] : st[(size_t)(i + n) * p.channels + c];
    }
  }
}

#define CV_THREADS 128
#define CV_CHUNK 16

__device__ __forceinline__ void unpack8(const uint4& raw, float (&f)[8]) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const float2 v = __bfloat1622float2(h[k]);
    f[2 * k] = v.x;
    f[2 * k + 1] = v.y;
  }
}
__device__ __forceinline__ uint4 pack8(const float (&f)[8]) {
  uint4 raw;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int k = 0; k < 4; ++k) h[k] = __floats2bfloat162_rn(f[2 * k], f[2 * k + 1]);
  return raw;
}

template <int TAPS>
__global__ void __launch_bounds__(CV_THREADS) conv_qkv_vec_kernel(ConvQkvParams p) {
  extern __shared__ float2 cs_sn[];                       // [CV_CHUNK][rot_dims / 2]
  const int c = (blockIdx.x * CV_THREADS + threadIdx.x) * 8;
  const bool live = c < p.channels;
  float w[TAPS][8];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {                        // constant data: fetched before the kernel ahead has finished
#pragma unroll
    for (int k = 0; k < 8; ++k) w[j][k] = 1.f;
    if (live && p.w != nullptr) {
      const float4* src = reinterpret_cast<const float4*>(p.w + (size_t)j * p.channels + c);
      const float4 a = src[0], b = src[1];
      w[j][0] = a.x; w[j][1] = a.y; w[j][2] = a.z; w[j][3] = a.w; w[j][4] = b.x; w[j][5] = b.y; w[j][6] = b.z; w[j][7] = b.w;
    }
  }
  pdl_trigger();
  pdl_wait();
  const int req = blockIdx.y;
  const int q0 = p.q_start[req], q1 = p.q_start[req + 1];
  const int t_lo = q0 + blockIdx.z * CV_CHUNK, t_hi = min(q1, t_lo + CV_CHUNK);
  if (t_lo >= q1) return;
  const int pairs = p.inv_freq != nullptr ? p.rot_dims >> 1 : 0;
  if (pairs > 0 && blockIdx.x * CV_THREADS * 8 < p.v0) {
    for (int i = threadIdx.x; i < (t_hi - t_lo) * pairs; i += CV_THREADS) {
      const int t = i / pairs, k = i - t * pairs;
      float2 v;
      turn((double)p.positions[t_lo + t], p.inv_freq[k], p.mult, v.x, v.y);
      cs_sn[t * pairs + k] = v;
    }
  }
  __syncthreads();
  if (!live) return;
  const int side = c < p.k0 ? 0 : (c < p.v0 ? 1 : 2);
  const int hd = side == 2 ? p.hd_v : p.hd;
  const int e = c - (side == 0 ? 0 : (side == 1 ? p.k0 : p.v0));
  const int h = e / hd, d = e - h * hd;
  const int pair0 = d >> 1;                               // the thread's four pairs; those from `pairs` on do not turn
  const int n_turn = side == 2 ? 0 : max(0, min(4, pairs - pair0));
  const bf16* x = (const bf16*)p.x + c;
  const int slot = p.slots != nullptr ? IE_SLOT(p.slots[req]) : -1;
  bf16* st = (slot >= 0 && p.state != nullptr && TAPS > 1) ? (bf16*)p.state + (size_t)slot * p.state_stride + c : nullptr;
  uint4 hist[TAPS > 1 ? TAPS - 1 : 1];                    // the last inputs, oldest first
#pragma unroll
  for (int i = 0; i < TAPS - 1; ++i) {
    const int src = t_lo - (TAPS - 1) + i;
    hist[i] = make_uint4(0u, 0u, 0u, 0u);
    if (src >= q0) hist[i] = *reinterpret_cast<const uint4*>(x + (size_t)src * p.x_stride);
    else if (st != nullptr) hist[i] = *reinterpret_cast<const uint4*>(st + (size_t)(TAPS - 1 - (q0 - src)) * p.channels);
  }
  constexpr int U = 4;                                    // rows on their way together
  for (int tb = t_lo; tb < t_hi; tb += U) {
    uint4 raw[U], kept[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      raw[u] = kept[u] = make_uint4(0u, 0u, 0u, 0u);
      if (tb + u < t_hi) {
        raw[u] = *reinterpret_cast<const uint4*>(x + (size_t)(tb + u) * p.x_stride);
        if (side == 2 && p.v_mode == 2)
          kept[u] = *reinterpret_cast<const uint4*>((const bf16*)p.v_kept + (size_t)(tb + u) * p.kv_heads * hd + e);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int t = tb + u;
      if (t >= t_hi) break;
      float y[8], f[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) y[k] = 0.f;
#pragma unroll
      for (int i = 0; i < TAPS - 1; ++i) {
        unpack8(hist[i], f);
#pragma unroll
        for (int k = 0; k < 8; ++k) y[k] = fmaf(w[i][k], f[k], y[k]);
      }
      unpack8(raw[u], f);
#pragma unroll
      for (int k = 0; k < 8; ++k) y[k] = fmaf(w[TAPS - 1][k], f[k], y[k]);
#pragma unroll
      for (int i = 0; i + 1 < TAPS - 1; ++i) hist[i] = hist[i + 1];
      if (TAPS > 1) hist[TAPS > 1 ? TAPS - 2 : 0] = raw[u];
      if (n_turn > 0) {
        const float2* row = cs_sn + (t - t_lo) * pairs + pair0;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          if (k < n_turn) {
            const float2 a = row[k];
            const float u0 = y[2 * k], v0 = y[2 * k + 1];
            y[2 * k] = fmaf(u0, a.x, -v0 * a.y);
            y[2 * k + 1] = fmaf(v0, a.x, u0 * a.y);
          }
        }
      }
      if (side == 0) {
        *reinterpret_cast<uint4*>((bf16*)p.q_out + (size_t)t * p.q_stride + e) = pack8(y);
        continue;
      }
      const int page_slot = p.slot_mapping != nullptr ? IE_SLOT(p.slot_mapping[t]) : -1;
      if (side == 2 && p.v_mode == 1)
        *reinterpret_cast<uint4*>((bf16*)p.v_kept + (size_t)t * p.kv_heads * hd + e) = pack8(y);
      if (side == 2 && p.v_mode == 2) {
        unpack8(kept[u], f);
#pragma unroll
        for (int k = 0; k < 8; ++k) y[k] = fmaf(p.lambda, f[k], (1.f - p.lambda) * y[k]);
      }
      bf16* pool = (bf16*)(side == 1 ? p.kpool : p.vpool);
      if (page_slot >= 0 && pool != nullptr)
        *reinterpret_cast<uint4*>(pool + (((size_t)(page_slot / p.page_size) * p.kv_heads + h) * p.page_size +
                                          page_slot % p.page_size) * hd + d) = pack8(y);
    }
  }
  if constexpr (TAPS > 1) {
    if (blockIdx.z > 0 || st == nullptr || !p.write_state) return;
    // the new state: what the registers hold when this chunk was all of the request, else the request's last inputs (a
    // chunk holds more tokens than there are taps, so those are all the step's own)
#pragma unroll
    for (int i = 0; i < TAPS - 1; ++i) {
      uint4 v = hist[i];
      if (t_hi < q1) v = *reinterpret_cast<const uint4*>(x + (size_t)(q1 - (TAPS - 1) + i) * p.x_stride);
      *reinterpret_cast<uint4*>(st + (size_t)i * p.channels) = v;
    }
  }
}

extern "C" int ie_conv_qkv(const void* x, int x_stride, const float* w, void* state, long long state_stride, int channels,
                           int taps, void* q_out, int q_stride, void* kpool, void* vpool, void* v_kept, int v_mode,
                           float lambda, const double* inv_freq, int rot_dims, int neighbours, float mult,
                           const int* positions, const int* slot_mapping, const int* q_start, const int* slots,
                           int n_requests, int heads, int kv_heads, int hd, int hd_v, int k0, int v0, int page_size,
                           int write_state, int act_dtype, int max_q_len, cudaStream_t stream) {
  if (n_requests <= 0 || max_q_len <= 0) return IE_OK;
  if (taps < 1 || taps > CQ_MAX_TAPS || heads <= 0 || kv_heads <= 0 || hd <= 0 || hd_v <= 0 || page_size <= 0) return IE_BAD_SIZE;
  if (w == nullptr && taps != 1) return IE_BAD_SIZE;
  if (rot_dims < 0 || (rot_dims & 1) || rot_dims > hd) return IE_BAD_SIZE;
  if (k0 < heads * hd || v0 < k0 + kv_heads * hd || channels < v0 + kv_heads * hd_v || x_stride < channels) return IE_BAD_SIZE;
  if (v_mode < 0 || v_mode > 2 || (v_mode && v_kept == nullptr)) return IE_BAD_SIZE;
  ConvQkvParams p;
  p.x = x; p.x_stride = x_stride; p.w = w; p.state = state; p.state_stride = state_stride; p.channels = channels; p.taps = taps;
  p.q_out = q_out; p.q_stride = q_stride; p.kpool = kpool; p.vpool = vpool; p.v_kept = v_kept; p.v_mode = v_mode;
  p.lambda = lambda; p.inv_freq = rot_dims > 0 ? inv_freq : nullptr; p.rot_dims = rot_dims; p.neighbours = neighbours;
  p.mult = mult; p.positions = positions; p.slot_mapping = slot_mapping; p.q_start = q_start; p.slots = slots;
  p.heads = heads; p.kv_heads = kv_heads; p.hd = hd; p.hd_v = hd_v; p.k0 = k0; p.v0 = v0; p.page_size = page_size;
  p.write_state = write_state;
  const uintptr_t at = (uintptr_t)x | (uintptr_t)w | (uintptr_t)state | (uintptr_t)q_out | (uintptr_t)kpool | (uintptr_t)vpool |
                       (uintptr_t)v_kept;
  const bool vec = act_dtype == IE_BF16 && taps <= CQ_VEC_TAPS && (hd % 8) == 0 && (hd_v % 8) == 0 && (channels % 8) == 0 &&
                   (k0 == heads * hd) && (v0 == k0 + kv_heads * hd) && (channels == v0 + kv_heads * hd_v) &&
                   (x_stride % 8) == 0 && (q_stride % 8) == 0 && (state_stride % 8) == 0 && (at & 15) == 0 &&
                   (rot_dims == 0 || neighbours);
  if (vec) {
    const int chunks = (max_q_len + CV_CHUNK - 1) / CV_CHUNK;
    if (chunks > 65535 || n_requests > 65535) return IE_BAD_SIZE;
    dim3 grid((channels / 8 + CV_THREADS - 1) / CV_THREADS, n_requests, chunks);
    const size_t smem = sizeof(float2) * CV_CHUNK * (size_t)(rot_dims >> 1);
    switch (taps) {
#define CV_GO(N) case N: return launch_k(conv_qkv_vec_kernel<N>, grid, CV_THREADS, smem, stream, p)
      CV_GO(1); CV_GO(2); CV_GO(3); CV_GO(4); CV_GO(5); CV_GO(6); CV_GO(7); CV_GO(8);
#undef CV_GO
    }
  }
  const int chunks = (max_q_len + CQ_CHUNK - 1) / CQ_CHUNK;
  if (chunks > 65535 || n_requests > 65535) return IE_BAD_SIZE;
  dim3 grid(heads + 2 * kv_heads, n_requests, chunks), block(32, CQ_TL);
  if (act_dtype == IE_F32) return launch_k(conv_qkv_kernel<float>, grid, block, 0, stream, p);
  if (act_dtype == IE_BF16) return launch_k(conv_qkv_kernel<bf16>, grid, block, 0, stream, p);
  return IE_BAD_DTYPE;
}

IE_CHECK_API(convqkv)

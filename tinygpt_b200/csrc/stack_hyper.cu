// stack_hyper.cu — hyper-connected blocks as plain kernels: any width, 1 … kMaxStreams copies, storage type T = bf16 or fp32.
// Every kernel starts with griddepcontrol.launch_dependents + griddepcontrol.wait (programmatic dependent launch).
#include "stack_hyper.cuh"

#include <algorithm>

namespace b200 {

namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ T cvt(float v);
template <> __device__ __forceinline__ float cvt<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 cvt<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) tot += red[i];
  __syncthreads();
  return tot;
}

template <int V> struct Vec;
template <> struct Vec<1> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[1]) { v[0] = *p; }
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
  static __device__ __forceinline__ void store(float* p, const float (&v)[1]) { *p = v[0]; }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct Vec<4> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  }
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    v[0] = bf16_lo(a.x); v[1] = bf16_hi(a.x); v[2] = bf16_lo(a.y); v[3] = bf16_hi(a.y);
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack2(v[0], v[1]), pack2(v[2], v[3]));
  }
};

// h and the token-shift mixes of row t, channel c; n(j) hands out the normed row j positions back (zeros before the sequence)
template <typename T, typename F>
__device__ __forceinline__ void conv_channel(const InputConv& c, int64_t t, int64_t n_tok, int width, int i, F&& n) {
  const float cur = n(0);
  float h = cur, hp = 0.f;
  if (c.w != nullptr)
    for (int j = 0; j < c.taps; ++j) h = fmaf(c.w[(int64_t)(c.taps - 1 - j) * width + i], n(j), h);
  if (c.h != nullptr) static_cast<T*>(c.h)[t * width + i] = cvt<T>(h);
  if (c.mu == nullptr) return;
  hp = n(1);
  if (c.w != nullptr)
    for (int j = 0; j < c.taps; ++j) hp = fmaf(c.w[(int64_t)(c.taps - 1 - j) * width + i], n(j + 1), hp);
#pragma unroll
  for (int s = 0; s < kShiftMixes; ++s)
    static_cast<T*>(c.mix)[(s * n_tok + t) * width + i] = cvt<T>(fmaf(hp - h, c.mu[(int64_t)s * width + i], h));
}

// The same for V neighbouring channels and compile-time taps, from a window n[0 … TAPS] of rows (n[j] = the row j positions back):
// the row h leaves with is handed out, hp is the row before's (only read with mu).
template <int TAPS, int V>
__device__ __forceinline__ void conv_window(const float (&n)[TAPS + 1][V], const float (&w)[TAPS][V], int from, float (&h)[V]) {
#pragma unroll
  for (int k = 0; k < V; ++k) {
    float a = n[from][k];
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      if (from + j <= TAPS) a = fmaf(w[TAPS - 1 - j][k], n[from + j][k], a);
    h[k] = a;
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_conv(const InputConv& c, int64_t t, int64_t n_tok, int width, int i, const float (&h)[V],
                                           const float (&hp)[V], const float (&mu)[kShiftMixes][V]) {
  if (c.h != nullptr) Vec<V>::store(static_cast<T*>(c.h) + t * width + i, h);
  if (c.mu == nullptr) return;
#pragma unroll
  for (int s = 0; s < kShiftMixes; ++s) {
    float m[V];
#pragma unroll
    for (int k = 0; k < V; ++k) m[k] = fmaf(hp[k] - h[k], mu[s][k], h[k]);
    Vec<V>::store(static_cast<T*>(c.mix) + (s * n_tok + t) * width + i, m);
  }
}
// the taps and blend weights of V channels
template <int TAPS, int V>
__device__ __forceinline__ void load_conv(const InputConv& c, int width, int i, float (&w)[TAPS][V], float (&mu)[kShiftMixes][V]) {
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    if (c.w != nullptr) {
      Vec<V>::load(c.w + (int64_t)j * width + i, w[j]);
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) w[j][k] = 0.f;
    }
  }
#pragma unroll
  for (int s = 0; s < kShiftMixes; ++s) {
    if (c.mu != nullptr) {
      Vec<V>::load(c.mu + (int64_t)s * width + i, mu[s]);
    } else {
#pragma unroll
      for (int k = 0; k < V; ++k) mu[s][k] = 0.f;
    }
  }
}

// One CTA per row; the row's u sits in shared memory between the sum of squares and the norm (a thread comes back to its own
// entries, so nothing but the sum crosses threads).  CT > 0: the convolution's taps, known at compile time (0: any number, or no
// convolution).
template <typename T, int S, int V, int CT>
__global__ void __launch_bounds__(512) hyper_step_kernel(const HyperStep p) {
  pdl_trigger();
  extern __shared__ float u[];
  __shared__ float red[32], c_in[S], c_out[S], c_mix[S * S];
  const int t = blockIdx.x, W = p.width, ns = p.streams;
  for (int e = threadIdx.x; e < S * S; e += blockDim.x) {   // weights: readable ahead of the wait
    const int s = e / S, d = e % S;
    c_mix[e] = s < ns && d < ns ? (p.prev.mix != nullptr ? p.prev.mix[s * ns + d] : s == d ? 1.f : 0.f) : 0.f;
    if (e < S) {
      c_in[e] = e < ns ? (p.in != nullptr ? p.in[e] : 1.f) : 0.f;
      c_out[e] = e < ns ? p.mult * (p.prev.out != nullptr ? p.prev.out[e] : 1.f) : 0.f;
    }
  }
  pdl_wait();
  __syncthreads();
  float* xr = p.x + (int64_t)t * ns * W;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    float xs[S][V], acc[V];
#pragma unroll
    for (int s = 0; s < S; ++s) {
      if (s < ns) {
        Vec<V>::load(xr + (int64_t)s * W + i, xs[s]);
      } else {
#pragma unroll
        for (int k = 0; k < V; ++k) xs[s][k] = 0.f;
      }
    }
    if (p.y != nullptr) {
      float yv[V], xn[S][V];
      if (p.y_bf16) Vec<V>::load(static_cast<const __nv_bfloat16*>(p.y) + (int64_t)t * W + i, yv);
      else Vec<V>::load(static_cast<const float*>(p.y) + (int64_t)t * W + i, yv);
#pragma unroll
      for (int d = 0; d < S; ++d) {
#pragma unroll
        for (int k = 0; k < V; ++k) {
          float a = c_out[d] * yv[k];
#pragma unroll
          for (int s = 0; s < S; ++s) a = fmaf(c_mix[s * S + d], xs[s][k], a);
          xn[d][k] = a;
        }
      }
#pragma unroll
      for (int s = 0; s < S; ++s) {
        if (s < ns) Vec<V>::store(xr + (int64_t)s * W + i, xn[s]);
#pragma unroll
        for (int k = 0; k < V; ++k) xs[s][k] = xn[s][k];
      }
    }
#pragma unroll
    for (int k = 0; k < V; ++k) {
      float a = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) a = fmaf(c_in[s], xs[s][k], a);
      acc[k] = a;
      ss += a * a;
    }
    Vec<V>::store(u + i, acc);
  }
  float inv = 1.f;
  if (p.norm_w != nullptr) inv = 1.f / sqrtf(block_sum(ss, red) / (float)W + p.eps);
  const int64_t row = (int64_t)t * W;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    float n[V];
    Vec<V>::load(u + i, n);
    if (p.norm_w != nullptr) {
      float w[V];
      Vec<V>::load(p.norm_w + i, w);
#pragma unroll
      for (int k = 0; k < V; ++k) n[k] = n[k] * inv * (p.offset + w[k]);
    }
    if (p.h != nullptr) Vec<V>::store(static_cast<T*>(p.h) + row + i, n);
    if (p.hn != nullptr) Vec<V>::store(p.hn + row + i, n);
    if (!p.conv) continue;
    // the row is its sequence's only new one: earlier rows come from the slot, which moves on at once
    if constexpr (CT > 0) {
      float* st = p.c.state + (int64_t)p.slot[t] * p.c.slot_stride + i;
      const int ps = p.pos[t];
      float win[CT + 1][V], w[CT][V], mu[kShiftMixes][V], h[V], hp[V];
#pragma unroll
      for (int j = 1; j <= CT; ++j) {
        if (ps - j >= 0) {
          Vec<V>::load(st + (int64_t)(CT - j) * W, win[j]);
        } else {
#pragma unroll
          for (int k = 0; k < V; ++k) win[j][k] = 0.f;
        }
      }
      load_conv<CT, V>(p.c, W, i, w, mu);
#pragma unroll
      for (int k = 0; k < V; ++k) win[0][k] = n[k];
      conv_window<CT, V>(win, w, 0, h);
      conv_window<CT, V>(win, w, 1, hp);
      store_conv<T, V>(p.c, t, p.n_tok, W, i, h, hp, mu);
#pragma unroll
      for (int e = 0; e < CT; ++e) Vec<V>::store(st + (int64_t)e * W, win[CT - 1 - e]);
      continue;
    }
    float* st = p.c.state + (int64_t)p.slot[t] * p.c.slot_stride;
    const int taps = p.c.taps, ps = p.pos[t];
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const int c = i + k;
      auto back = [&](int j) { return j == 0 ? n[k] : ps - j >= 0 ? st[(int64_t)(taps - j) * W + c] : 0.f; };
      conv_channel<T>(p.c, t, p.n_tok, W, c, back);
      for (int e = 0; e < taps; ++e) {   // entry e: the row taps − 1 − e positions back; always further along than what is written
        const float v = back(taps - 1 - e);
        st[(int64_t)e * W + c] = v;
      }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128) hyper_embed_kernel(float* __restrict__ x, const T* __restrict__ embed,
                                                          const int32_t* __restrict__ tok, int vocab, int width, int streams,
                                                          float scale) {
  pdl_trigger();
  pdl_wait();
  int id = tok[blockIdx.x];
  if (id < 0 || id >= vocab) id = 0;
  const T* row = embed + (int64_t)id * width;
  float* xr = x + (int64_t)blockIdx.x * streams * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float v = ldf<T>(row + i) * scale;
    for (int s = 0; s < streams; ++s) xr[(int64_t)s * width + i] = v;
  }
}

template <typename T>
__global__ void __launch_bounds__(256) input_conv_kernel(const InputConv c, const float* __restrict__ hn, const int32_t* __restrict__ slot,
                                                         const int32_t* __restrict__ pos, int n_tok, int width) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, i = blockIdx.y * 256 + threadIdx.x;
  if (i >= width) return;
  const int front = rows_in_front(slot, pos, t, c.taps), ps = pos[t];
  const float* st = c.state + (int64_t)slot[t] * c.slot_stride;
  auto back = [&](int j) {
    if (j <= front) return hn[(int64_t)(t - j) * width + i];
    return ps - j >= 0 ? st[(int64_t)(c.taps - (j - front)) * width + i] : 0.f;   // j − front rows before the step's first one
  };
  conv_channel<T>(c, t, n_tok, width, i, back);
}

// The same for kConvStrip rows per CTA and V neighbouring channels per thread: while a sequence goes on, the window slides through
// registers and a row's h is the next row's hp.
constexpr int kConvStrip = 8;
template <typename T, int TAPS, int V>
__global__ void __launch_bounds__(128) input_conv_strip_kernel(const InputConv c, const float* __restrict__ hn, const int32_t* __restrict__ slot,
                                                               const int32_t* __restrict__ pos, int n_tok, int width) {
  pdl_trigger();
  const int t0 = blockIdx.x * kConvStrip, i = (blockIdx.y * 128 + threadIdx.x) * V;
  const bool live = i < width;
  float w[TAPS][V], mu[kShiftMixes][V];
  if (live) load_conv<TAPS, V>(c, width, i, w, mu);
  pdl_wait();
  if (!live) return;
  float win[TAPS + 1][V], h[V], hp[V];
  const int t1 = min(t0 + kConvStrip, n_tok);
  const bool one = rows_one_seq(slot, pos, t0, t1);
#pragma unroll 2
  for (int t = t0; t < t1; ++t) {
    if (t == t0 || (!one && !row_same_seq(slot, pos, t, 1))) {   // a window of its own: the step's rows in front, then the slot's
      const int front = rows_in_front(slot, pos, t, TAPS), ps = pos[t];
      const float* st = c.state + (int64_t)slot[t] * c.slot_stride + i;
#pragma unroll
      for (int j = 1; j <= TAPS; ++j) {
        if (j <= front) {
          Vec<V>::load(hn + (int64_t)(t - j) * width + i, win[j]);
        } else if (ps - j >= 0) {
          Vec<V>::load(st + (int64_t)(TAPS - (j - front)) * width, win[j]);
        } else {
#pragma unroll
          for (int k = 0; k < V; ++k) win[j][k] = 0.f;
        }
      }
      conv_window<TAPS, V>(win, w, 1, hp);
    } else {
#pragma unroll
      for (int j = TAPS; j > 0; --j)
#pragma unroll
        for (int k = 0; k < V; ++k) win[j][k] = win[j - 1][k];
#pragma unroll
      for (int k = 0; k < V; ++k) hp[k] = h[k];
    }
    Vec<V>::load(hn + (int64_t)t * width + i, win[0]);
    conv_window<TAPS, V>(win, w, 0, h);
    store_conv<T, V>(c, t, n_tok, width, i, h, hp, mu);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) shift_state_kernel(const ShiftState p) {
  pdl_trigger();
  pdl_wait();
  const ShiftSource& s = p.src[blockIdx.z];
  const int c = blockIdx.y * 256 + threadIdx.x;
  if (c >= s.channels) return;
  const int r0 = p.seg_row0[blockIdx.x], cnt = p.seg_count[blockIdx.x], last = r0 + cnt - 1, ps = p.pos[last];
  float* st = s.state + (int64_t)p.slot[r0] * p.slot_stride;
  for (int e = 0; e < s.keep; ++e) {
    const int j = s.keep - 1 - e;   // positions back from the last row
    float v = 0.f;
    if (j < cnt) {
      const int64_t o = (int64_t)(last - j) * s.ld + c;
      v = s.f32 ? static_cast<const float*>(s.rows)[o] : ldf<T>(static_cast<const T*>(s.rows) + o);
    } else if (ps - j >= 0) {
      v = st[(int64_t)(e + cnt) * s.channels + c];   // an old entry, further along than anything written so far
    }
    st[(int64_t)e * s.channels + c] = v;
  }
}

}  // namespace

#define HYPER_DTYPE_CHECK(dtype) \
  B200_CHECK_ARG((dtype) == B200_BF16 || (dtype) == B200_F32, "stack op: unknown dtype %d", (int)(dtype))

// four neighbouring channels at a time (the caller checks that the width is a multiple of four)
static bool conv_vec_ok(const InputConv& c) {
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  return al(c.w) && al(c.mu) && al(c.h) && al(c.mix) && al(c.state) && c.slot_stride % 4 == 0;   // null pointers are aligned
}

int launch_hyper_step(const HyperStep& p, int dtype, cudaStream_t st) {
  HYPER_DTYPE_CHECK(dtype);
  B200_CHECK_ARG(p.x && p.n_tok > 0 && p.width > 0 && p.streams >= 1 && p.streams <= kMaxStreams,
                 "hyper step: bad arguments (1 … %d streams)", kMaxStreams);
  B200_CHECK_ARG(p.streams == 1 || ((p.y == nullptr || (p.prev.out && p.prev.mix))), "hyper step: several streams need their weights");
  B200_CHECK_ARG(!p.conv || (p.c.state && p.slot && p.pos && p.c.taps >= 1 && (p.c.h || p.c.mix)), "hyper step: incomplete convolution");
  const size_t smem = (size_t)p.width * 4;
  B200_CHECK_ARG(smem <= 200 * 1024, "hyper step: rows wider than 51200 are not built");
  auto al = [](const void* q, size_t a) { return (reinterpret_cast<uintptr_t>(q) % a) == 0; };
  const bool vec = p.width % 4 == 0 && al(p.x, 16) && (p.y == nullptr || al(p.y, 16)) && (p.h == nullptr || al(p.h, 16)) &&
                   (p.hn == nullptr || al(p.hn, 16)) && (p.norm_w == nullptr || al(p.norm_w, 16)) &&
                   (!p.conv || (conv_vec_ok(p.c) && p.c.taps <= 4));
  // few rows: as many threads as there are entries, one round of loads; many rows: 256 threads
  const int items = vec ? p.width / 4 : p.width;
  const int threads = p.n_tok <= 148 && items > 256 ? 512 : 256;
#define B200_HS(T, S, V, CT)                                                                                            \
  do {                                                                                                              \
    static bool attr_done = false;                                                                                  \
    if (smem > 40 * 1024 && !attr_done) {                                                                           \
      B200_CUDA(cudaFuncSetAttribute(hyper_step_kernel<T, S, V, CT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); \
      attr_done = true;                                                                                             \
    }                                                                                                               \
    B200_CUDA(launch_pdl(hyper_step_kernel<T, S, V, CT>, dim3(p.n_tok), dim3(threads), smem, st, stack_pdl(), p));       \
  } while (0)
#define B200_HS_S(T, V, CT)                        \
  do {                                             \
    if (p.streams == 1) B200_HS(T, 1, V, CT);      \
    else if (p.streams == 2) B200_HS(T, 2, V, CT); \
    else if (p.streams <= 4) B200_HS(T, 4, V, CT); \
    else B200_HS(T, 8, V, CT);                     \
  } while (0)
#define B200_HS_T(T)                                \
  do {                                              \
    if (!vec) B200_HS_S(T, 1, 0);                   \
    else if (!p.conv) B200_HS_S(T, 4, 0);           \
    else if (p.c.taps == 1) B200_HS_S(T, 4, 1);     \
    else if (p.c.taps == 2) B200_HS_S(T, 4, 2);     \
    else if (p.c.taps == 3) B200_HS_S(T, 4, 3);     \
    else B200_HS_S(T, 4, 4);                        \
  } while (0)
  if (dtype == B200_F32) B200_HS_T(float);
  else B200_HS_T(__nv_bfloat16);
#undef B200_HS_T
#undef B200_HS_S
#undef B200_HS
  return B200_OK;
}

int launch_hyper_embed(float* x, const void* embed, const int32_t* tok, int64_t n_tok, int vocab, int width, int streams, float scale,
                       int dtype, cudaStream_t st) {
  HYPER_DTYPE_CHECK(dtype);
  B200_CHECK_ARG(x && embed && tok && n_tok > 0 && width > 0 && streams > 0, "hyper embed: bad arguments");
  if (dtype == B200_F32)
    B200_CUDA(launch_pdl(hyper_embed_kernel<float>, dim3((unsigned)n_tok), dim3(128), 0, st, stack_pdl(), x, (const float*)embed, tok,
                         vocab, width, streams, scale));
  else
    B200_CUDA(launch_pdl(hyper_embed_kernel<__nv_bfloat16>, dim3((unsigned)n_tok), dim3(128), 0, st, stack_pdl(), x,
                         (const __nv_bfloat16*)embed, tok, vocab, width, streams, scale));
  return B200_OK;
}

int launch_input_conv(const InputConv& c, const float* hn, const int32_t* slot, const int32_t* pos, int n_tok, int width, int dtype,
                      cudaStream_t st) {
  HYPER_DTYPE_CHECK(dtype);
  B200_CHECK_ARG(hn && slot && pos && c.state && n_tok > 0 && width > 0 && c.taps >= 1 && c.taps <= kConvMaxTaps && (c.h || c.mix) &&
                     (c.mu == nullptr || c.mix),
                 "input convolution: bad arguments (1 … %d taps)", kConvMaxTaps);
  if (width % 4 == 0 && c.taps <= 4 && conv_vec_ok(c) && (reinterpret_cast<uintptr_t>(hn) & 15) == 0) {
    const dim3 grid((n_tok + kConvStrip - 1) / kConvStrip, (width / 4 + 127) / 128);
#define B200_IC(T, TAPS) B200_CUDA(launch_pdl(input_conv_strip_kernel<T, TAPS, 4>, grid, dim3(128), 0, st, stack_pdl(), c, hn, slot, pos, n_tok, width))
#define B200_IC_T(T)                    \
  do {                                  \
    if (c.taps == 1) B200_IC(T, 1);     \
    else if (c.taps == 2) B200_IC(T, 2); \
    else if (c.taps == 3) B200_IC(T, 3); \
    else B200_IC(T, 4);                 \
  } while (0)
    if (dtype == B200_F32) B200_IC_T(float);
    else B200_IC_T(__nv_bfloat16);
#undef B200_IC_T
#undef B200_IC
    return B200_OK;
  }
  const dim3 grid(n_tok, (width + 255) / 256);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(input_conv_kernel<float>, grid, dim3(256), 0, st, stack_pdl(), c, hn, slot, pos, n_tok, width));
  else B200_CUDA(launch_pdl(input_conv_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, stack_pdl(), c, hn, slot, pos, n_tok, width));
  return B200_OK;
}

int launch_shift_state(const ShiftState& p, int dtype, cudaStream_t st) {
  HYPER_DTYPE_CHECK(dtype);
  if (p.n_src == 0) return B200_OK;
  B200_CHECK_ARG(p.seg_row0 && p.seg_count && p.slot && p.pos && p.n_seg > 0 && p.n_src <= kShiftSources, "shift state: bad arguments");
  int ch = 1;
  for (int i = 0; i < p.n_src; ++i) {
    B200_CHECK_ARG(p.src[i].rows && p.src[i].state && p.src[i].channels > 0 && p.src[i].keep >= 0, "shift state: bad source");
    ch = std::max(ch, p.src[i].channels);
  }
  const dim3 grid(p.n_seg, (ch + 255) / 256, p.n_src);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(shift_state_kernel<float>, grid, dim3(256), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(shift_state_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, stack_pdl(), p));
  return B200_OK;
}

}  // namespace b200

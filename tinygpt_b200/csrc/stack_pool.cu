// stack_pool.cu — attention with pooled blocks and mixed heads as plain kernels: any head counts and sizes, storage type
// T = bf16 or fp32.  Every kernel starts with griddepcontrol.launch_dependents + griddepcontrol.wait.
#include "stack_pool.cuh"

#include <algorithm>

#include "stack_hyper.cuh"

namespace b200 {

namespace {

template <typename T> __device__ __forceinline__ float ldf(const T* p);
template <> __device__ __forceinline__ float ldf<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ldf<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
template <typename T> __device__ __forceinline__ T cvt(float v);
template <> __device__ __forceinline__ float cvt<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 cvt<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// What one CTA of the preparation works on: key/value head g, query heads [h0, h0 + nh) of those that read it, and — in the first
// CTA of the group — key head and value head g.  Its channels, in order: [nh·dk: q | dk: k | dv: v].
struct PrepUnit {
  int g, h0, nh, nq, mine;
  bool kv;
};
__device__ __forceinline__ PrepUnit prep_unit(const PoolAttn& p, int y) {
  const int per = p.a.heads / p.a.kv_heads, hc = p.heads_per_cta, nc = (per + hc - 1) / hc;
  PrepUnit u;
  u.g = y / nc;
  const int first = (y % nc) * hc;
  u.h0 = u.g * per + first;
  u.nh = min(hc, per - first);
  u.nq = u.nh * p.a.dim;
  u.kv = first == 0 && !p.q_only;
  u.mine = u.nq + (u.kv ? p.a.dim + p.a.vdim : 0);
  return u;
}
// the projection column of the CTA's e-th channel
__device__ __forceinline__ int prep_col(const PoolAttn& p, const PrepUnit& u, int e) {
  const int dk = p.a.dim, dv = p.a.vdim;
  return e < u.nq ? p.off_q + u.h0 * dk + e : e < u.nq + dk ? p.off_k + u.g * dk + (e - u.nq) : p.off_v + u.g * dv + (e - u.nq - dk);
}

// One warp: the norm of one head's convolved channels x, the turn of its first rot_dims entries, and the row it leaves: a query's
// in q, or a key's cache row.  A key's entries stay in x as the cache holds them.
template <typename T>
__device__ __forceinline__ void finish_head(const PoolAttn& p, int ps, bool key, float* x, T* dst, int lane) {
  const int dk = p.a.dim, half = p.d.rot_dims / 2;
  const float* tab = half > 0 ? p.d.rot_table + (int64_t)ps * half * 2 : nullptr;
  const float* w = key ? p.d.k_norm : p.d.q_norm;
  float inv = 1.f;
  if (w != nullptr) {
    float ss = 0.f;
    for (int i = lane; i < dk; i += 32) ss += x[i] * x[i];
    inv = 1.f / sqrtf(warp_sum(ss) / (float)dk + p.eps);
  }
  for (int i = lane; i < dk - half; i += 32) {   // half pairs, then the entries that do not turn
    if (i < half) {
      const int i0 = p.d.rot_interleaved ? 2 * i : i, i1 = p.d.rot_interleaved ? 2 * i + 1 : i + half;
      float u = x[i0] * inv, v = x[i1] * inv;
      if (w != nullptr) {
        u *= w[i0];
        v *= w[i1];
      }
      const float c = tab[2 * i], s = tab[2 * i + 1];
      const T a = cvt<T>(u * c - v * s), b = cvt<T>(v * c + u * s);
      dst[i0] = a;
      dst[i1] = b;
      if (key) {
        x[i0] = ldf<T>(&a);
        x[i1] = ldf<T>(&b);
      }
    } else {
      float u = x[i + half] * inv;
      if (w != nullptr) u *= w[i + half];
      const T a = cvt<T>(u);
      dst[i + half] = a;
      if (key) x[i + half] = ldf<T>(&a);
    }
  }
}

// One CTA per (token, PrepUnit).  The convolution of every channel goes to shared memory; then one warp per query / key head takes
// the head's norm and turns its first rot_dims entries.  Queries leave for q, keys and values for the slot's cache rows.
template <typename T>
__global__ void __launch_bounds__(256) pool_prep_kernel(const PoolAttn p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];   // [nh·dk: q | dk: k | dv: v]
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const PrepUnit un = prep_unit(p, blockIdx.y);
  const int H = p.a.heads, G = p.a.kv_heads, dk = p.a.dim, dv = p.a.vdim, g = un.g, taps = p.d.conv_w != nullptr ? p.d.taps : 1;
  const int nq = un.nq, mine = un.mine, ps = p.pos[t];
  const T* row = static_cast<const T*>(p.proj) + (int64_t)t * p.ld_proj;
  float* cs = p.conv_state + (int64_t)p.slot[t] * p.conv_slot_stride;
  const int front = p.single ? 0 : rows_in_front(p.slot, p.pos, t, taps - 1);
  for (int e = tid; e < mine; e += 256) {
    const int col = prep_col(p, un, e);
    auto back = [&](int j) {
      if (j <= front) return ldf<T>(row - (int64_t)j * p.ld_proj + col);
      return ps - j >= 0 ? cs[(int64_t)(taps - 1 - (j - front)) * p.ld_proj + col] : 0.f;
    };
    float acc = back(0);
    if (p.d.conv_w != nullptr) {
      acc = 0.f;
      for (int j = 0; j < taps; ++j) acc = fmaf(p.d.conv_w[(int64_t)(taps - 1 - j) * p.ld_proj + col], back(j), acc);
      if (p.single)
        for (int i = 0; i < taps - 1; ++i) {   // entry i: the row taps − 2 − i positions back, further along than what is written
          const float v = back(taps - 2 - i);
          cs[(int64_t)i * p.ld_proj + col] = v;
        }
    }
    sm[e] = acc;
  }
  __syncthreads();
  T* kc = static_cast<T*>(p.kcache) + (int64_t)p.slot[t] * p.k_slot_stride;
  T* vc = static_cast<T*>(p.vcache) + (int64_t)p.slot[t] * p.v_slot_stride;
  for (int hh = warp; hh < un.nh + (un.kv ? 1 : 0); hh += 8) {
    const bool key = hh == un.nh;
    finish_head<T>(p, ps, key, sm + hh * dk, key ? kc + ((int64_t)ps * G + g) * dk : static_cast<T*>(p.q) + ((int64_t)t * H + un.h0 + hh) * dk, lane);
  }
  if (!un.kv) return;
  float* v = sm + nq + dk;
  for (int i = tid; i < dv; i += 256) {
    const T a = cvt<T>(v[i]);
    vc[((int64_t)ps * G + g) * dv + i] = a;
    v[i] = ldf<T>(&a);
  }
  if (!p.single || p.d.pool <= 0 || (ps + 1) % p.d.pool != 0) return;
  __syncthreads();
  const int P = p.d.pool, b = ps / P;
  const float inv = 1.f / (float)P;
  for (int e = tid; e < dk + dv; e += 256) {   // the block's earlier rows were cached by earlier steps
    const bool key = e < dk;
    const int n = key ? dk : dv, i = key ? e : e - dk;
    T* c = key ? kc : vc;
    float s = 0.f;
    for (int j = 0; j < P - 1; ++j) s += ldf<T>(c + ((int64_t)(b * P + j) * G + g) * n + i);
    s += sm[nq + e];
    c[((int64_t)(p.max_ctx + b) * G + g) * n + i] = cvt<T>(s * inv);
  }
}

// Prompts: kPrepStrip tokens per CTA; while a sequence goes on, a channel's window slides through registers.
constexpr int kPrepStrip = 8;
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) pool_prep_strip_kernel(const PoolAttn p) {
  pdl_trigger();
  extern __shared__ float sm[];   // [kPrepStrip][nh·dk: q | dk: k | dv: v]
  const int t0 = blockIdx.x * kPrepStrip, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const PrepUnit un = prep_unit(p, blockIdx.y);
  const int H = p.a.heads, G = p.a.kv_heads, dk = p.a.dim, dv = p.a.vdim, g = un.g;
  const int nq = un.nq, mine = un.mine, n = min(kPrepStrip, p.n_tok - t0);
  pdl_wait();
  const bool one = rows_one_seq(p.slot, p.pos, t0, t0 + n);
  for (int e = tid; e < mine; e += 256) {
    const int col = prep_col(p, un, e);
    const T* x = static_cast<const T*>(p.proj) + (int64_t)t0 * p.ld_proj + col;
    float w[TAPS], win[TAPS];   // win[j]: the row j positions back
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = p.d.conv_w[(int64_t)j * p.ld_proj + col];
    for (int r = 0; r < n; ++r) {
      const int t = t0 + r;
      if (r == 0 || (!one && !row_same_seq(p.slot, p.pos, t, 1))) {
        const int front = rows_in_front(p.slot, p.pos, t, TAPS - 1), ps = p.pos[t];
        const float* cs = p.conv_state + (int64_t)p.slot[t] * p.conv_slot_stride + col;
#pragma unroll
        for (int j = 1; j < TAPS; ++j)
          win[j] = j <= front ? ldf<T>(x + (int64_t)(r - j) * p.ld_proj) : ps - j >= 0 ? cs[(int64_t)(TAPS - 1 - (j - front)) * p.ld_proj] : 0.f;
      } else {
#pragma unroll
        for (int j = TAPS - 1; j > 0; --j) win[j] = win[j - 1];
      }
      win[0] = ldf<T>(x + (int64_t)r * p.ld_proj);
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(w[TAPS - 1 - j], win[j], acc);
      sm[r * mine + e] = acc;
    }
  }
  __syncthreads();
  const int rows = un.nh + (un.kv ? 1 : 0);
  for (int u = warp; u < n * rows; u += 8) {
    const int r = u / rows, hh = u % rows, t = t0 + r, ps = p.pos[t];
    const bool key = hh == un.nh;
    T* kc = static_cast<T*>(p.kcache) + (int64_t)p.slot[t] * p.k_slot_stride;
    finish_head<T>(p, ps, key, sm + r * mine + hh * dk, key ? kc + ((int64_t)ps * G + g) * dk : static_cast<T*>(p.q) + ((int64_t)t * H + un.h0 + hh) * dk,
                   lane);
  }
  if (!un.kv) return;
  for (int r = warp; r < n; r += 8) {
    const int t = t0 + r;
    T* vd = static_cast<T*>(p.vcache) + (int64_t)p.slot[t] * p.v_slot_stride + ((int64_t)p.pos[t] * G + g) * dv;
    for (int i = lane; i < dv; i += 32) vd[i] = cvt<T>(sm[r * mine + nq + dk + i]);
  }
}

// The same preparation without shared memory, for bf16 rows whose head sizes are multiples of four up to 128 and whose pairs are
// neighbours: one warp per (strip of tokens, head), a lane holds four neighbouring channels.  The strip's rows are requested
// together; a token then costs the convolution in registers, one warp sum for the norm, the turn inside the lane and one
// eight-byte store.  single: a strip is one row, whose convolution state — requested ahead of the dependency wait, an earlier step
// left it there — moves on here.
constexpr int kHeadStrip = 4;
template <int TAPS, bool SINGLE>
__global__ void __launch_bounds__(256, 4) head_prep_kernel(const PoolAttn p) {
  using T = __nv_bfloat16;
  constexpr int STRIP = SINGLE ? 1 : kHeadStrip;
  pdl_trigger();
  const int H = p.a.heads, G = p.a.kv_heads, unit = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (unit >= H + (p.q_only ? 0 : 2 * G)) return;
  const bool is_q = unit < H, is_v = unit >= H + G;
  const int head = is_q ? unit : is_v ? unit - H - G : unit - H, ch = is_v ? p.a.vdim : p.a.dim, c = lane * 4;
  const bool act = c < ch;
  const int col = (is_q ? p.off_q : is_v ? p.off_v : p.off_k) + head * ch + (act ? c : 0);
  const int t0 = blockIdx.x * STRIP, n = min(STRIP, p.n_tok - t0);
  float w[TAPS][4], nw[4] = {1.f, 1.f, 1.f, 1.f}, win[TAPS][4];   // win[j]: the row j positions back
  auto load4 = [](float(&o)[4], const float* q) {
    const float4 v = *reinterpret_cast<const float4*>(q);
    o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
  };
#pragma unroll
  for (int j = 0; j < TAPS; ++j) load4(w[j], p.d.conv_w + (int64_t)j * p.ld_proj + col);
  const float* norm_w = is_v ? nullptr : is_q ? p.d.q_norm : p.d.k_norm;
  if (norm_w != nullptr && act) load4(nw, norm_w + c);
  float* cs = p.conv_state + col;   // the slot's part is added below
  if constexpr (SINGLE) {
    cs += (int64_t)p.slot[t0] * p.conv_slot_stride;
    const int ps = p.pos[t0];
#pragma unroll
    for (int j = 1; j < TAPS; ++j) {
      if (ps - j >= 0) load4(win[j], cs + (int64_t)(TAPS - 1 - j) * p.ld_proj);
      else win[j][0] = win[j][1] = win[j][2] = win[j][3] = 0.f;
    }
  }
  pdl_wait();
  const T* x = static_cast<const T*>(p.proj) + (int64_t)t0 * p.ld_proj + col;
  uint2 raw[STRIP];
#pragma unroll
  for (int r = 0; r < STRIP; ++r) raw[r] = r < n ? *reinterpret_cast<const uint2*>(x + (int64_t)r * p.ld_proj) : make_uint2(0, 0);
  auto unpack4 = [](float(&o)[4], uint2 v) {
    o[0] = bf16_lo(v.x); o[1] = bf16_hi(v.x); o[2] = bf16_lo(v.y); o[3] = bf16_hi(v.y);
  };
  const bool one = SINGLE || rows_one_seq(p.slot, p.pos, t0, t0 + n);
  const float inv_n = 1.f / (float)ch;
#pragma unroll
  for (int r = 0; r < STRIP; ++r) {
    if (r >= n) break;
    const int t = t0 + r, ps = p.pos[t];
    if constexpr (!SINGLE) {
      if (r == 0 || (!one && !row_same_seq(p.slot, p.pos, t, 1))) {
        const int front = rows_in_front(p.slot, p.pos, t, TAPS - 1);
        const float* st = cs + (int64_t)p.slot[t] * p.conv_slot_stride;
#pragma unroll
        for (int j = 1; j < TAPS; ++j) {
          if (j <= front) unpack4(win[j], *reinterpret_cast<const uint2*>(x + (int64_t)(r - j) * p.ld_proj));
          else if (ps - j >= 0) load4(win[j], st + (int64_t)(TAPS - 1 - (j - front)) * p.ld_proj);
          else win[j][0] = win[j][1] = win[j][2] = win[j][3] = 0.f;
        }
      } else {
#pragma unroll
        for (int j = TAPS - 1; j > 0; --j)
#pragma unroll
          for (int i = 0; i < 4; ++i) win[j][i] = win[j - 1][i];
      }
    }
    unpack4(win[0], raw[r]);
    float y[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      y[i] = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) y[i] = fmaf(w[TAPS - 1 - j][i], win[j][i], y[i]);
    }
    if (norm_w != nullptr) {
      const float ss = warp_sum(act ? fmaf(y[0], y[0], fmaf(y[1], y[1], fmaf(y[2], y[2], y[3] * y[3]))) : 0.f);
      const float inv = 1.f / sqrtf(ss * inv_n + p.eps);
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] *= inv * nw[i];
    }
    if (!is_v && c < p.d.rot_dims) {   // two pairs; their {cos, sin} lie side by side
      float cs4[4];
      load4(cs4, p.d.rot_table + (int64_t)ps * p.d.rot_dims + c);
#pragma unroll
      for (int i = 0; i < 4; i += 2) {
        const float a = y[i], b = y[i + 1];
        y[i] = a * cs4[i] - b * cs4[i + 1];
        y[i + 1] = b * cs4[i] + a * cs4[i + 1];
      }
    }
    if (act) {
      T* dst = is_q ? static_cast<T*>(p.q) + ((int64_t)t * H + head) * ch
                    : (is_v ? static_cast<T*>(p.vcache) + (int64_t)p.slot[t] * p.v_slot_stride
                            : static_cast<T*>(p.kcache) + (int64_t)p.slot[t] * p.k_slot_stride) + ((int64_t)ps * G + head) * ch;
      *reinterpret_cast<uint2*>(dst + c) = make_uint2(pack2(y[0], y[1]), pack2(y[2], y[3]));
      if constexpr (SINGLE) {
#pragma unroll
        for (int i = 0; i < TAPS - 1; ++i)   // entry i: the row TAPS − 2 − i positions back
          *reinterpret_cast<float4*>(cs + (int64_t)i * p.ld_proj) =
              make_float4(win[TAPS - 2 - i][0], win[TAPS - 2 - i][1], win[TAPS - 2 - i][2], win[TAPS - 2 - i][3]);
      }
    }
  }
}
// what head_prep_kernel takes
bool head_prep_ok(const PoolAttn& p, int dtype) {
  const b200_attn_desc& a = p.a;
  auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };   // null pointers are aligned
  return dtype == B200_BF16 && p.d.conv_w != nullptr && p.d.taps <= 4 && !(p.single && p.d.pool > 0) && a.dim % 4 == 0 && a.dim <= 128 &&
         a.vdim % 4 == 0 && a.vdim <= 128 && p.d.rot_dims % 4 == 0 && (p.d.rot_dims == 0 || p.d.rot_interleaved) && p.off_q % 4 == 0 &&
         p.off_k % 4 == 0 && p.off_v % 4 == 0 && p.ld_proj % 4 == 0 && p.k_slot_stride % 4 == 0 && p.v_slot_stride % 4 == 0 &&
         p.conv_slot_stride % 4 == 0 && al(p.proj) && al(p.q) && al(p.kcache) && al(p.vcache) && al(p.conv_state) && al(p.d.conv_w) &&
         al(p.d.q_norm) && al(p.d.k_norm) && al(p.d.rot_table);
}

// The blocks whose last position is among a sequence's rows of this step: the means of their cached keys and values (rows of
// this step or of earlier ones).
template <typename T>
__global__ void __launch_bounds__(256) pool_blocks_kernel(const PoolAttn p) {
  pdl_trigger();
  pdl_wait();
  const int t = p.seg_row0[blockIdx.z], P = p.d.pool, ps = p.pos[t], b = ps / P + blockIdx.x;
  if (b >= (ps + p.seg_count[blockIdx.z]) / P) return;
  const int nk = p.a.kv_heads * p.a.dim, nv = p.a.kv_heads * p.a.vdim, e = blockIdx.y * 256 + threadIdx.x;
  if (e >= nk + nv) return;
  const bool key = e < nk;
  const int n = key ? nk : nv, i = key ? e : e - nk;
  T* c = key ? static_cast<T*>(p.kcache) + (int64_t)p.slot[t] * p.k_slot_stride : static_cast<T*>(p.vcache) + (int64_t)p.slot[t] * p.v_slot_stride;
  float s = 0.f;
#pragma unroll 8
  for (int j = 0; j < P; ++j) s += ldf<T>(c + (int64_t)(b * P + j) * n + i);
  c[(int64_t)(p.max_ctx + b) * n + i] = cvt<T>(s * (1.f / (float)P));
}

__device__ __forceinline__ float capped(float s, float cap) { return cap > 0.f ? cap * tanhf(s / cap) : s; }

// One CTA of eight warps per (row, split of the key list): the capped scores of every head, and each head's running maximum and
// sum over the split.  A warp takes one key per lane and up to kPoolHC query heads of one key/value head at a time: the key row's
// entries are loaded once for all of them, the queries come from shared memory.
constexpr int kPoolHC = 4;
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) pool_scores_kernel(const PoolAttn p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float qs[];   // [H·dk]
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int H = p.a.heads, G = p.a.kv_heads, dk = p.a.dim, per = H / G, i = p.pos[t];
  const int lo = pool_lo(i, p.a.window), nb = pool_nb(i, p.a.window, p.d.pool), total = nb + i - lo + 1;
  const int begin = blockIdx.y * p.keys_per_split, end = min(total, begin + p.keys_per_split);
  if (begin >= end) return;
  const T* q = static_cast<const T*>(p.q) + (int64_t)t * H * dk;
  for (int e = threadIdx.x; e < H * dk; e += 256) qs[e] = ldf<T>(q + e) * p.a.scale;
  __syncthreads();
  const T* K = static_cast<const T*>(p.kcache) + (int64_t)p.slot[t] * p.k_slot_stride;
  const int chunks = (per + kPoolHC - 1) / kPoolHC;
  for (int un = warp; un < G * chunks; un += 8) {
    const int g = un / chunks, h0 = g * per + (un % chunks) * kPoolHC, nh = min(kPoolHC, (g + 1) * per - h0);
    float m[kPoolHC], l[kPoolHC];
#pragma unroll
    for (int u = 0; u < kPoolHC; ++u) {
      m[u] = -INFINITY;
      l[u] = 0.f;
    }
    for (int k0 = begin; k0 < end; k0 += 32) {
      const int idx = k0 + lane;
      if (idx < end) {
        const int r = idx < nb ? p.max_ctx + idx : lo + (idx - nb);
        const T* kr = K + ((int64_t)r * G + g) * dk;
        float s[kPoolHC];
#pragma unroll
        for (int u = 0; u < kPoolHC; ++u) s[u] = 0.f;
        if constexpr (VEC) {   // sixteen-byte pieces of the key row, eight requested together
          const uint4* k4 = reinterpret_cast<const uint4*>(kr);
          for (int d0 = 0; d0 < dk >> 3; d0 += 8) {
            uint4 kq[8];
#pragma unroll
            for (int w = 0; w < 8; ++w) kq[w] = d0 + w < (dk >> 3) ? k4[d0 + w] : make_uint4(0, 0, 0, 0);
#pragma unroll
            for (int w = 0; w < 8; ++w) {
              if (d0 + w >= (dk >> 3)) break;
              float kf[8];
              unpack8(kq[w], kf);
#pragma unroll
              for (int u = 0; u < kPoolHC; ++u) {
                if (u < nh) {
                  const float* qq = qs + (h0 + u) * dk + (d0 + w) * 8;
#pragma unroll
                  for (int x = 0; x < 8; ++x) s[u] = fmaf(qq[x], kf[x], s[u]);
                }
              }
            }
          }
        } else {
          for (int d = 0; d < dk; ++d) {
            const float kv = ldf<T>(kr + d);
#pragma unroll
            for (int u = 0; u < kPoolHC; ++u)
              if (u < nh) s[u] = fmaf(qs[(h0 + u) * dk + d], kv, s[u]);
          }
        }
#pragma unroll
        for (int u = 0; u < kPoolHC; ++u) {
          if (u < nh) {
            const float v = capped(s[u], p.d.softcap);
            p.scores[((int64_t)t * H + h0 + u) * p.nk_max + idx] = v;
            const float mn = fmaxf(m[u], v);
            l[u] = l[u] * expf(m[u] - mn) + expf(v - mn);   // first key: exp(−inf) = 0
            m[u] = mn;
          }
        }
      }
    }
#pragma unroll
    for (int u = 0; u < kPoolHC; ++u) {
      if (u >= nh) break;
      const float mt = warp_max(m[u]);
      const float lt = warp_sum(m[u] == -INFINITY ? 0.f : l[u] * expf(m[u] - mt));
      if (lane == 0) {
        float* o = p.parts + (((int64_t)t * H + h0 + u) * p.nsplit + blockIdx.y) * 2;
        o[0] = mt;
        o[1] = lt;
      }
    }
  }
}

// One CTA per (row, split): every head's maximum and denominator over all splits (and the sink), then tile by tile of
// kPoolTile keys the weights of all heads, their mix, and the weighted values — a thread owns value columns and the query heads
// that read them; the sums over tiles sit in shared memory.
template <typename T, int VC>
__global__ void __launch_bounds__(256) pool_values_kernel(const PoolAttn p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = p.a.heads, G = p.a.kv_heads, dv = p.a.vdim, per = H / G, i = p.pos[t];
  constexpr int KP = kPoolTile + 1;
  float* s_m = sm;                    // [H]
  float* s_il = s_m + H;              // [H]
  float* s_w = s_il + H;              // [H][KP]
  float* s_x = s_w + H * KP;          // [H][KP] mixed
  float* s_o = s_x + H * KP;          // [H·dv]
  const int lo = pool_lo(i, p.a.window), nb = pool_nb(i, p.a.window, p.d.pool), total = nb + i - lo + 1;
  const int begin = blockIdx.y * p.keys_per_split, end = min(total, begin + p.keys_per_split);
  if (begin >= end) return;
  const int live = (total + p.keys_per_split - 1) / p.keys_per_split;   // splits that hold keys
  for (int h = warp; h < H; h += 8) {
    const float* o = p.parts + ((int64_t)t * H + h) * p.nsplit * 2;
    float m = p.d.sink != nullptr ? p.d.sink[h] : -INFINITY;
    for (int s = lane; s < live; s += 32) m = fmaxf(m, o[2 * s]);
    m = warp_max(m);
    float l = 0.f;
    for (int s = lane; s < live; s += 32) l += o[2 * s + 1] * expf(o[2 * s] - m);
    l = warp_sum(l);
    if (p.d.sink != nullptr) l += expf(p.d.sink[h] - m);
    if (lane == 0) {
      s_m[h] = m;
      s_il[h] = 1.f / l;
    }
  }
  for (int e = tid; e < H * dv; e += 256) s_o[e] = 0.f;
  __syncthreads();
  const T* V = static_cast<const T*>(p.vcache) + (int64_t)p.slot[t] * p.v_slot_stride;
  for (int k0 = begin; k0 < end; k0 += kPoolTile) {
    const int n = min(kPoolTile, end - k0);
    for (int h = warp; h < H; h += 8)
      s_w[h * KP + lane] = lane < n ? expf(p.scores[((int64_t)t * H + h) * p.nk_max + k0 + lane] - s_m[h]) * s_il[h] : 0.f;
    __syncthreads();
    const float* wm = s_w;
    if (p.d.talk != nullptr) {
      for (int h = warp; h < H; h += 8) {
        const float* T0 = p.d.talk + (int64_t)h * H;
        float a = 0.f;
        for (int g = 0; g < H; ++g) a = fmaf(T0[g], s_w[g * KP + lane], a);
        s_x[h * KP + lane] = a;
      }
      wm = s_x;
      __syncthreads();
    }
    const int cols = G * dv / VC;
    for (int e = tid; e < cols; e += 256) {
      const int c = e * VC, g = c / dv, cc = c % dv;   // VC columns of one head (dv is a multiple of VC)
      for (int u0 = 0; u0 < per; u0 += kPoolHC) {
        const int nh = min(kPoolHC, per - u0), h0 = g * per + u0;
        float acc[kPoolHC][VC];
#pragma unroll
        for (int u = 0; u < kPoolHC; ++u)
#pragma unroll
          for (int x = 0; x < VC; ++x) acc[u][x] = 0.f;
#pragma unroll 8
        for (int k = 0; k < n; ++k) {
          const int idx = k0 + k, r = idx < nb ? p.max_ctx + idx : lo + (idx - nb);
          const T* vr = V + ((int64_t)r * G) * dv + c;
          float v[VC];
          if constexpr (VC == 2) {
            const uint32_t b = *reinterpret_cast<const uint32_t*>(vr);
            v[0] = bf16_lo(b);
            v[1] = bf16_hi(b);
          } else {
            v[0] = ldf<T>(vr);
          }
#pragma unroll
          for (int u = 0; u < kPoolHC; ++u) {
            if (u < nh) {
              const float w = wm[(h0 + u) * KP + k];
#pragma unroll
              for (int x = 0; x < VC; ++x) acc[u][x] = fmaf(w, v[x], acc[u][x]);
            }
          }
        }
#pragma unroll
        for (int u = 0; u < kPoolHC; ++u)
          if (u < nh)
#pragma unroll
            for (int x = 0; x < VC; ++x) s_o[(h0 + u) * dv + cc + x] += acc[u][x];
      }
    }
    __syncthreads();
  }
  if (p.nsplit > 1) {
    float* o = p.outs + ((int64_t)t * p.nsplit + blockIdx.y) * H * dv;
    for (int e = tid; e < H * dv; e += 256) o[e] = s_o[e];
    return;
  }
  T* y = static_cast<T*>(p.mid) + (int64_t)t * p.ld_mid;
  for (int e = tid; e < max(H * dv, p.n_pad); e += 256) y[e] = cvt<T>(e < H * dv ? s_o[e] * p.out_scale : 0.f);
}

template <typename T>
__global__ void __launch_bounds__(128) pool_merge_kernel(const PoolAttn p) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, e = blockIdx.y * 128 + threadIdx.x, n = p.a.heads * p.a.vdim, i = p.pos[t];
  if (e >= max(n, p.n_pad)) return;
  const int total = pool_nb(i, p.a.window, p.d.pool) + i - pool_lo(i, p.a.window) + 1;
  const int live = (total + p.keys_per_split - 1) / p.keys_per_split;
  float a = 0.f;
  if (e < n) {
    const float* o = p.outs + (int64_t)t * p.nsplit * n + e;
#pragma unroll 8
    for (int s = 0; s < live; ++s) a += o[(int64_t)s * n];
  }
  static_cast<T*>(p.mid)[(int64_t)t * p.ld_mid + e] = cvt<T>(a * p.out_scale);
}

int check_pool(const PoolAttn& p) {
  const b200_attn_desc& a = p.a;
  B200_CHECK_ARG(a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.vdim > 0 && a.window >= 0 && p.d.pool >= 0,
                 "pool attention: bad sizes (heads %d, kv_heads %d, dim %d, vdim %d)", a.heads, a.kv_heads, a.dim, a.vdim);
  B200_CHECK_ARG(p.d.rot_dims >= 0 && p.d.rot_dims % 2 == 0 && p.d.rot_dims <= a.dim && (p.d.rot_dims == 0 || p.d.rot_table),
                 "pool attention: rot_dims %d must be even, at most the head size %d, with a table", p.d.rot_dims, a.dim);
  B200_CHECK_ARG(p.q_only || (p.d.q_norm == nullptr) == (p.d.k_norm == nullptr), "pool attention: one of the two head norms is missing");
  B200_CHECK_ARG(p.d.softcap >= 0.f, "pool attention: negative softcap");
  B200_CHECK_ARG(p.q && p.kcache && p.vcache && p.slot && p.pos && p.n_tok > 0 && p.max_ctx > 0, "pool attention: null argument");
  return B200_OK;
}

}  // namespace

#define POOL_DTYPE_CHECK(dtype) \
  B200_CHECK_ARG((dtype) == B200_BF16 || (dtype) == B200_F32, "stack op: unknown dtype %d", (int)(dtype))

int launch_pool_prep(const PoolAttn& run, int dtype, cudaStream_t st) {
  POOL_DTYPE_CHECK(dtype);
  PoolAttn p = run;
  int rc = check_pool(p);
  if (rc != B200_OK) return rc;
  B200_CHECK_ARG(p.proj != nullptr, "pool attention: null projection");
  B200_CHECK_ARG(p.d.conv_w == nullptr || (p.d.taps >= 1 && p.d.taps <= kConvMaxTaps && (p.d.taps == 1 || p.conv_state)),
                 "pool attention: 1 … %d convolution taps with a state", kConvMaxTaps);
  if (head_prep_ok(p, dtype)) {
    const dim3 hg((p.n_tok + (p.single ? 1 : kHeadStrip) - 1) / (p.single ? 1 : kHeadStrip), (p.a.heads + (p.q_only ? 0 : 2 * p.a.kv_heads) + 7) / 8);
#define B200_HP(TAPS)                                                                                                   \
  do {                                                                                                                  \
    if (p.single) B200_CUDA(launch_pdl(head_prep_kernel<TAPS, true>, hg, dim3(256), 0, st, stack_pdl(), p));            \
    else B200_CUDA(launch_pdl(head_prep_kernel<TAPS, false>, hg, dim3(256), 0, st, stack_pdl(), p));                    \
  } while (0)
    if (p.d.taps == 1) B200_HP(1);
    else if (p.d.taps == 2) B200_HP(2);
    else if (p.d.taps == 3) B200_HP(3);
    else B200_HP(4);
#undef B200_HP
    return B200_OK;
  }
  // query heads per CTA: the strip's channels within 48 KB, and few rows spread over many CTAs
  const int per = p.a.heads / p.a.kv_heads, dk = p.a.dim, kv = p.q_only ? 0 : dk + p.a.vdim, limit = 12 * 1024;   // floats
  B200_CHECK_ARG(dk + kv <= limit, "pool attention: one query head and one key/value head exceed %d channels", limit);
  const bool strips = !p.single && p.n_tok > kPrepStrip && p.d.conv_w != nullptr && p.d.taps <= 4 && kPrepStrip * (dk + kv) <= limit;
  const int fit = ((strips ? limit / kPrepStrip : limit) - kv) / dk;
  p.heads_per_cta = std::max(1, std::min({per, fit, p.n_tok <= 16 ? 4 : 8}));
  const size_t smem = (size_t)(p.heads_per_cta * dk + kv) * 4;
  const unsigned units = (unsigned)(p.a.kv_heads * ((per + p.heads_per_cta - 1) / p.heads_per_cta));
  if (strips) {
    const dim3 sg((p.n_tok + kPrepStrip - 1) / kPrepStrip, units);
#define B200_PP(T, TAPS) B200_CUDA(launch_pdl(pool_prep_strip_kernel<T, TAPS>, sg, dim3(256), kPrepStrip * smem, st, stack_pdl(), p))
#define B200_PP_T(T)                    \
  do {                                  \
    if (p.d.taps == 1) B200_PP(T, 1);   \
    else if (p.d.taps == 2) B200_PP(T, 2); \
    else if (p.d.taps == 3) B200_PP(T, 3); \
    else B200_PP(T, 4);                 \
  } while (0)
    if (dtype == B200_F32) B200_PP_T(float);
    else B200_PP_T(__nv_bfloat16);
#undef B200_PP_T
#undef B200_PP
    return B200_OK;
  }
  const dim3 grid(p.n_tok, units);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(pool_prep_kernel<float>, grid, dim3(256), smem, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(pool_prep_kernel<__nv_bfloat16>, grid, dim3(256), smem, st, stack_pdl(), p));
  return B200_OK;
}

int launch_pool_blocks(const PoolAttn& p, int dtype, cudaStream_t st) {
  POOL_DTYPE_CHECK(dtype);
  int rc = check_pool(p);
  if (rc != B200_OK) return rc;
  if (p.d.pool <= 0) return B200_OK;
  B200_CHECK_ARG(p.seg_row0 && p.seg_count && p.n_seg > 0 && p.max_count > 0, "pool blocks: null sequences");
  const dim3 bg(p.max_count / p.d.pool + 1, (p.a.kv_heads * (p.a.dim + p.a.vdim) + 255) / 256, p.n_seg);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(pool_blocks_kernel<float>, bg, dim3(256), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(pool_blocks_kernel<__nv_bfloat16>, bg, dim3(256), 0, st, stack_pdl(), p));
  return B200_OK;
}

int launch_pool_attention(const PoolAttn& p, int dtype, cudaStream_t st) {
  POOL_DTYPE_CHECK(dtype);
  int rc = check_pool(p);
  if (rc != B200_OK) return rc;
  const int H = p.a.heads, dk = p.a.dim, dv = p.a.vdim;
  B200_CHECK_ARG(p.scores && p.parts && p.mid && p.nk_max > 0 && p.nsplit >= 1 && p.nsplit <= kPoolMaxSplits && p.keys_per_split > 0 &&
                     (int64_t)p.nsplit * p.keys_per_split >= p.nk_max && (p.nsplit == 1 || p.outs),
                 "pool attention: bad workspace");
  const size_t sm_q = (size_t)H * dk * 4, sm_v = (size_t)(2 * H + 2 * H * (kPoolTile + 1) + H * dv) * 4;
  B200_CHECK_ARG(sm_q <= 200 * 1024 && sm_v <= 200 * 1024, "pool attention: heads · head size exceeds one CTA's shared memory");
  static bool attr_done = false;
  if (!attr_done) {
    B200_CUDA(cudaFuncSetAttribute(pool_scores_kernel<float, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    B200_CUDA(cudaFuncSetAttribute(pool_scores_kernel<__nv_bfloat16, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    B200_CUDA(cudaFuncSetAttribute(pool_scores_kernel<__nv_bfloat16, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    B200_CUDA(cudaFuncSetAttribute(pool_values_kernel<float, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    B200_CUDA(cudaFuncSetAttribute(pool_values_kernel<__nv_bfloat16, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    B200_CUDA(cudaFuncSetAttribute(pool_values_kernel<__nv_bfloat16, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    attr_done = true;
  }
  const dim3 grid(p.n_tok, p.nsplit);
  const bool kvec = dtype == B200_BF16 && dk % 8 == 0 && p.k_slot_stride % 8 == 0 && (reinterpret_cast<uintptr_t>(p.kcache) & 15) == 0;
  const bool vvec = dtype == B200_BF16 && dv % 2 == 0 && p.v_slot_stride % 2 == 0 && (reinterpret_cast<uintptr_t>(p.vcache) & 3) == 0;
  if (dtype == B200_F32) {
    B200_CUDA(launch_pdl(pool_scores_kernel<float, false>, grid, dim3(256), sm_q, st, stack_pdl(), p));
    B200_CUDA(launch_pdl(pool_values_kernel<float, 1>, grid, dim3(256), sm_v, st, stack_pdl(), p));
  } else {
    if (kvec) B200_CUDA(launch_pdl(pool_scores_kernel<__nv_bfloat16, true>, grid, dim3(256), sm_q, st, stack_pdl(), p));
    else B200_CUDA(launch_pdl(pool_scores_kernel<__nv_bfloat16, false>, grid, dim3(256), sm_q, st, stack_pdl(), p));
    if (vvec) B200_CUDA(launch_pdl(pool_values_kernel<__nv_bfloat16, 2>, grid, dim3(256), sm_v, st, stack_pdl(), p));
    else B200_CUDA(launch_pdl(pool_values_kernel<__nv_bfloat16, 1>, grid, dim3(256), sm_v, st, stack_pdl(), p));
  }
  if (p.nsplit > 1) {
    const dim3 mg(p.n_tok, (std::max(H * dv, p.n_pad) + 127) / 128);
    if (dtype == B200_F32) B200_CUDA(launch_pdl(pool_merge_kernel<float>, mg, dim3(128), 0, st, stack_pdl(), p));
    else B200_CUDA(launch_pdl(pool_merge_kernel<__nv_bfloat16>, mg, dim3(128), 0, st, stack_pdl(), p));
  }
  return B200_OK;
}

}  // namespace b200

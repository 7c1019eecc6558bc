// stack_rec.cu — mixers of post-norm blocks as plain kernels: the preparation of an attention mixer's projection rows, one
// scan for linear recurrences with a per-channel or per-head decay and an optional rank-one removal, the passes of the
// generalized delta rule and of Mamba-2 around it, and the post-norm that also leaves the next sublayer's operand copy.
// fp32 for norms, angles, gates, decays, step sizes, the recurrence and its state; storage type T = bf16 or fp32.
// Every kernel starts with griddepcontrol.launch_dependents + griddepcontrol.wait (programmatic dependent launch).
#include "stack_rec.cuh"

#include <algorithm>
#include <type_traits>

#include "stack_hyper.cuh"

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
__device__ __forceinline__ float sigmoidf(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float siluf(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplusf(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------------------------------------ attention preparation
// One CTA per token.  q and k: the sum of squares over the WHOLE projection (all heads), the weight of that entry, then the
// rotation of the first rot_dims entries of every head (entry i with entry i + rot_dims/2, or — rot_interleaved — entry 2i
// with entry 2i + 1).  v: every head by its own root
// mean square, then the mix with the kept values.  All in fp32 from the T-typed projection, written back as T once.
template <typename T>
__global__ void __launch_bounds__(256) attn_prep_kernel(const AttnPrep p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const int t = blockIdx.x, tid = threadIdx.x;
  const int H = p.a.heads, G = p.a.kv_heads, dk = p.a.dim, dv = p.a.vdim;
  const int half = p.d.rot_dims / 2, items = dk - half;   // per head: `half` pairs, then the entries from rot_dims on
  T* row = static_cast<T*>(p.proj) + (int64_t)t * p.ld_proj;
  const float* tab = half > 0 ? p.d.rot_table + (int64_t)p.pos[t] * half * 2 : nullptr;
  for (int which = 0; which < (p.q_only ? 1 : 2); ++which) {
    T* x = row + (which ? p.off_k : p.off_q);
    const int n = (which ? G : H) * dk, nh = which ? G : H;
    const float* w = which ? p.d.k_norm : p.d.q_norm;
    float inv = 1.f;
    if (p.d.qk_norm) {
      float ss = 0.f;
      for (int i = tid; i < n; i += 256) {
        const float v = ldf<T>(x + i);
        ss += v * v;
      }
      inv = 1.f / sqrtf(block_sum(ss, red) / (float)n + p.eps);
    }
    if (!p.d.qk_norm && half == 0) continue;
    for (int e = tid; e < nh * items; e += 256) {
      const int hd = e / items, j = e % items;
      if (j < half) {
        const int i0 = hd * dk + (p.d.rot_interleaved ? 2 * j : j), i1 = i0 + (p.d.rot_interleaved ? 1 : half);
        float a = ldf<T>(x + i0) * inv, b = ldf<T>(x + i1) * inv;
        if (p.d.qk_norm) {
          a *= w[i0];
          b *= w[i1];
        }
        const float c = tab[2 * j], s = tab[2 * j + 1];
        x[i0] = cvt<T>(a * c - b * s);
        x[i1] = cvt<T>(b * c + a * s);
      } else if (p.d.qk_norm) {
        const int i = hd * dk + j + half;
        x[i] = cvt<T>(ldf<T>(x + i) * inv * w[i]);
      }
    }
  }
  if ((!p.d.v_norm && p.d.v_mix == 0) || p.q_only) return;
  T* v = row + p.off_v;
  T* keep = p.vkeep != nullptr ? static_cast<T*>(p.vkeep) + (int64_t)t * p.ld_keep : nullptr;
  const float lam = p.d.v_mix == 2 ? p.d.mix_lambda[0] : 0.f;
  const int warp = tid >> 5, lane = tid & 31;
  for (int g = warp; g < G; g += 8) {
    float inv = 1.f;
    if (p.d.v_norm) {
      float ss = 0.f;
      for (int i = lane; i < dv; i += 32) {
        const float a = ldf<T>(v + g * dv + i);
        ss += a * a;
      }
      inv = 1.f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
    }
    for (int i = lane; i < dv; i += 32) {
      float a = ldf<T>(v + g * dv + i) * inv;
      if (p.d.v_mix == 2) a = (1.f - lam) * a + lam * ldf<T>(keep + g * dv + i);
      v[g * dv + i] = cvt<T>(a);
      if (p.d.v_mix == 1) keep[g * dv + i] = cvt<T>(a);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------ the scan
// With a removal: one warp per (sequence, head, NC value columns): lane l holds rows l, l + 32, … of its columns of S (DR rows per lane and
// column); 8·NC columns per CTA.  The CTA walks its sequence CH tokens at a time: the chunk's decay, key, query (and removal,
// unit key) rows (fp32, zero past dk) and the CTA's columns of v sit in shared memory, staged once for all eight warps,
// while the next chunk's values are already on their way into registers — the walk waits for memory once per sequence.  A
// token costs a warp the removal's dot with the OLD columns (warp sums the update waits for, NC side by side), DR
// multiply-adds per operand and column, and the output's dot with the NEW columns.  Columns never read each other, so
// the result of a sequence does not depend on what else is in the step; the order of the sums inside a column is fixed by
// dk alone (lane l sums rows l, l + 32, …, then the butterfly), whatever NC is.
template <int DR, int NC>
__global__ void __launch_bounds__(256, 2) lin_scan_kernel(const LinScan p) {
  pdl_trigger();
  pdl_wait();
  constexpr int DK = 32 * DR;
  // tokens per chunk: what 4 KB of one operand hold, 4 … 32 — the next chunk waits in registers, and two CTAs share an SM
  constexpr int CH0 = 1024 / DK;
  constexpr int CH = CH0 > 32 ? 32 : CH0 < 4 ? 4 : CH0;
  constexpr int NV = 5;                                   // staged vectors per token: d, b, r, p, q
  constexpr int NQ = CH * NV * DK / 256;                  // staged vector elements per thread and chunk
  constexpr int COLS = 8 * NC;
  constexpr int NVR = (CH * COLS + 255) / 256;            // staged values per thread and chunk
  __shared__ float s_x[CH][NV][DK];
  __shared__ float s_v[CH][COLS];
  const int seg = blockIdx.x, hd = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  const int dk = p.dk, dv = p.dv;
  const int j0 = blockIdx.z * COLS, jw = j0 + warp * NC;
  const int r0 = p.seg_row0 != nullptr ? p.seg_row0[seg] : seg;
  const int cnt = p.seg_count != nullptr ? p.seg_count[seg] : 1;
  float* st = p.state + (int64_t)p.slot[r0] * p.slot_stride + (int64_t)hd * dk * dv;
  const bool fresh = p.pos[r0] == 0;
  float S[NC][DR];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
#pragma unroll
    for (int i = 0; i < DR; ++i) {
      const int d = lane + 32 * i;
      S[c][i] = (jw + c < dv && !fresh && d < dk) ? st[(int64_t)d * dv + jw + c] : 0.f;
    }
  }
  const int hs = hd / p.share;   // the head whose b / r vectors this head reads
  const float* src_d = p.d_scalar ? p.d + hd : p.d + (int64_t)hd * dk;
  const float* src_b = p.b + (int64_t)hs * dk;
  const float* src_r = p.r + (int64_t)hs * dk;
  const float* src_p = p.p + (int64_t)hd * dk;
  const float* src_q = p.q + (int64_t)(p.q_shared ? hs : hd) * dk;
  float r_x[NQ], r_v[NVR];
  auto fetch = [&](int c0) {
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int e = tid + 256 * i, t = e / (NV * DK), w = (e / DK) % NV, d = e % DK;
      float val = 0.f;
      if (c0 + t < cnt && d < dk) {
        const int64_t base = (int64_t)(r0 + c0 + t) * p.ld;
        const float* src = w == 0 ? src_d : w == 1 ? src_b : w == 2 ? src_r : w == 3 ? src_p : src_q;
        val = src[base + ((w == 0 && p.d_scalar) ? 0 : d)];
      }
      r_x[i] = val;
    }
#pragma unroll
    for (int i = 0; i < NVR; ++i) {
      const int e = tid + 256 * i, t = e / COLS, c = j0 + e % COLS;
      float val = 0.f;
      if (e < CH * COLS && c0 + t < cnt && c < dv) {
        const int64_t base = (int64_t)(r0 + c0 + t) * p.ld;
        val = p.v[base + (int64_t)hd * dv + c];
        if (p.vscale != nullptr) val *= p.vscale[base + hd];
      }
      r_v[i] = val;
    }
  };
  fetch(0);
  for (int c0 = 0; c0 < cnt; c0 += CH) {
    const int n = min(CH, cnt - c0);
    __syncthreads();   // the previous chunk has been read
#pragma unroll
    for (int i = 0; i < NQ; ++i) (&s_x[0][0][0])[tid + 256 * i] = r_x[i];
#pragma unroll
    for (int i = 0; i < NVR; ++i)
      if (tid + 256 * i < CH * COLS) (&s_v[0][0])[tid + 256 * i] = r_v[i];
    __syncthreads();
    if (c0 + CH < cnt) fetch(c0 + CH);
    if (jw >= dv) continue;   // warps past the last column only help with the staging
    for (int t4 = 0; t4 < n; t4 += 4) {   // the outputs' warp sums of four tokens run side by side, off the state's chain
      float dot[4][NC];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int t = t4 + u;             // t < CH always (CH is a multiple of 4)
#pragma unroll
        for (int c = 0; c < NC; ++c) dot[u][c] = 0.f;
        if (t >= n) continue;             // rows past the chunk's end hold zeros: they must not touch the state
        float rem[NC], vj[NC];
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          rem[c] = 0.f;
          vj[c] = s_v[t][warp * NC + c];
        }
#pragma unroll
        for (int i = 0; i < DR; ++i) {
          const float qq = s_x[t][4][lane + 32 * i];
#pragma unroll
          for (int c = 0; c < NC; ++c) rem[c] = fmaf(qq, S[c][i], rem[c]);
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
          for (int c = 0; c < NC; ++c) rem[c] += __shfl_xor_sync(0xffffffffu, rem[c], o);
        }
#pragma unroll
        for (int i = 0; i < DR; ++i) {
          const int d = lane + 32 * i;
          const float dd = s_x[t][0][d], bb = s_x[t][1][d], rr = s_x[t][2][d], pp = s_x[t][3][d];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            const float sn = fmaf(bb, vj[c], fmaf(-pp, rem[c], dd * S[c][i]));
            S[c][i] = sn;
            dot[u][c] = fmaf(sn, rr, dot[u][c]);
          }
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
        for (int u = 0; u < 4; ++u) {
#pragma unroll
          for (int c = 0; c < NC; ++c) dot[u][c] += __shfl_xor_sync(0xffffffffu, dot[u][c], o);
        }
      }
      if (lane < 4 * NC) {                // lane u·NC + c hands out token t4 + u, column jw + c
        const int u = lane / NC, c = lane % NC;
        float mine = 0.f;
#pragma unroll
        for (int uu = 0; uu < 4; ++uu) {
#pragma unroll
          for (int cc = 0; cc < NC; ++cc) mine = (uu == u && cc == c) ? dot[uu][cc] : mine;
        }
        if (t4 + u < n && jw + c < dv) p.o[(int64_t)(r0 + c0 + t4 + u) * p.ld_o + (int64_t)hd * dv + jw + c] = mine;
      }
    }
  }
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    if (jw + c >= dv) continue;
#pragma unroll
    for (int i = 0; i < DR; ++i) {
      const int d = lane + 32 * i;
      if (d < dk) st[(int64_t)d * dv + jw + c] = S[c][i];
    }
  }
}

// Without a removal no row of S waits for another: a CTA of NT threads takes kScanCols value columns of one (sequence, head), a
// thread a tile of RS neighbouring rows and four neighbouring columns (an operand a thread reads from shared memory serves four
// multiply-adds: the walk is bound by that traffic).  A token's output parts meet inside a warp by four shuffles per thread and,
// once per chunk, over the warps through shared memory; nothing the state waits for.  The chunk's decay, key and query rows come
// in by cp.async while the chunk before is walked (two buffers).  The order of the sums inside a column is fixed by dk alone.
// MODE 0: d is the decay, 1: the decay minus one (a decay close to one keeps all its digits), 2: the decay minus one, and the
// output reads the columns BEFORE the token joins them, plus the token's bonus times its value.  SCALAR: one decay per head.
constexpr int kScanCols = 16;
template <int RS, int NT, bool SCALAR>
struct ScanCols {
  static constexpr int DK = NT / 4 * RS, NV = SCALAR ? 2 : 3;   // staged vectors per token: b, r (, d)
  static constexpr int CH0 = 2048 / DK, CH = CH0 > 32 ? 32 : CH0 < 4 ? 4 : CH0;
  static constexpr int smem = (2 * CH * NV * DK + CH * (NT / 32) * kScanCols + 2 * CH * (kScanCols + 2)) * 4;
};
__device__ __forceinline__ void scan_cp(float* dst, const float* src, int bytes, bool wide) {
  const uint32_t d = smem_u32(dst);
  if (wide) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(d), "l"(src), "r"(bytes) : "memory");
}
// two fp32 multiply-adds (products) in one instruction; a pair of neighbouring rows travels as one 64-bit register pair
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t pair2(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 split2(uint64_t a) {
  float2 d;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(a));
  return d;
}
template <int RS, int NT, int MODE, bool SCALAR>
__global__ void __launch_bounds__(NT, RS <= 8 ? 512 / NT : 2) lin_scan_cols_kernel(const LinScan p, const bool wide) {
  using C = ScanCols<RS, NT, SCALAR>;
  constexpr int DK = C::DK, NV = C::NV, CH = C::CH, NW = NT / 32, NVR = (CH * kScanCols + NT - 1) / NT;
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) float sm[];
  float* const s_x = sm;                               // [2][CH][NV][DK]
  float* const s_v = s_x + 2 * CH * NV * DK;           // [2][CH][kScanCols]
  float* const s_part = s_v + 2 * CH * kScanCols;      // [CH][NW][kScanCols]
  float* const s_s = s_part + CH * NW * kScanCols;      // [2][CH][2]: the token's scalar decay and bonus
  const int seg = blockIdx.x, hd = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int dk = p.dk, dv = p.dv, c4 = (tid & 3) * 4, j0 = blockIdx.z * kScanCols + c4, d0 = (tid >> 2) * RS;
  const int r0 = p.seg_row0 != nullptr ? p.seg_row0[seg] : seg;
  const int cnt = p.seg_count != nullptr ? p.seg_count[seg] : 1;
  float* st = p.state + (int64_t)p.slot[r0] * p.slot_stride + (int64_t)hd * dk * dv;
  const bool fresh = p.pos[r0] == 0;
  uint64_t S[RS / 2][4];
  auto held = [&](int i, int c) { return j0 + c < dv && d0 + i < dk; };
#pragma unroll
  for (int i = 0; i < RS / 2; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c)
      S[i][c] = pair2(!fresh && held(2 * i, c) ? st[(int64_t)(d0 + 2 * i) * dv + j0 + c] : 0.f,
                      !fresh && held(2 * i + 1, c) ? st[(int64_t)(d0 + 2 * i + 1) * dv + j0 + c] : 0.f);
  const int hs = hd / p.share;   // the head whose b / r vectors this head reads
  const float* src_b = p.b + (int64_t)hs * dk;
  const float* src_r = p.r + (int64_t)hs * dk;
  const float* src_d = SCALAR ? p.d + hd : p.d + (int64_t)hd * dk;
  auto stage = [&](int c0, int buf) {
    const int n = min(CH, cnt - c0);
    float* x = s_x + buf * (CH * NV * DK);
    if (wide) {   // a thread keeps its place in the row and takes every RP-th token
      constexpr int UN = DK / 4, RP = NT / UN;
      const int td = (tid % UN) * 4, tr = tid / UN, bytes = td < dk ? 16 : 0;   // zeros past the key size
      const int64_t o = (int64_t)(r0 + c0 + tr) * p.ld + (td < dk ? td : 0), ld = p.ld * RP;
      const float *qb = src_b + o, *qr = src_r + o, *qd = SCALAR ? nullptr : src_d + o;
      float* dst = x + tr * (NV * DK) + td;
#pragma unroll
      for (int u = 0; u < (CH + RP - 1) / RP; ++u) {
        if (tr + u * RP >= n) break;
        scan_cp(dst + u * RP * NV * DK, qb + u * ld, bytes, true);
        scan_cp(dst + u * RP * NV * DK + DK, qr + u * ld, bytes, true);
        if constexpr (!SCALAR) scan_cp(dst + u * RP * NV * DK + 2 * DK, qd + u * ld, bytes, true);
      }
    } else {
      for (int e = tid; e < n * NV * DK; e += NT) {
        const int t = e / (NV * DK), w = (e / DK) % NV, d = e % DK;
        const float* src = (w == 0 ? src_b : w == 1 ? src_r : src_d) + (int64_t)(r0 + c0 + t) * p.ld;
        scan_cp(x + e, d < dk ? src + d : src, d < dk ? 4 : 0, false);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float r_v[NVR], r_s[2];
  auto fetch = [&](int c0) {
#pragma unroll
    for (int i = 0; i < NVR; ++i) {
      const int e = tid + NT * i, t = e / kScanCols, c = blockIdx.z * kScanCols + e % kScanCols;
      float val = 0.f;
      if (t < CH && c0 + t < cnt && c < dv) {
        const int64_t base = (int64_t)(r0 + c0 + t) * p.ld;
        val = p.v[base + (int64_t)hd * dv + c];
        if (p.vscale != nullptr) val *= p.vscale[base + hd];
      }
      r_v[i] = val;
    }
    const bool live = tid < CH && c0 + tid < cnt;
    if constexpr (SCALAR) r_s[0] = live ? src_d[(int64_t)(r0 + c0 + tid) * p.ld] : 0.f;
    if constexpr (MODE == 2) r_s[1] = live ? p.bonus[(int64_t)(r0 + c0 + tid) * p.ld + hd] : 0.f;
  };
  stage(0, 0);
  fetch(0);
  for (int c0 = 0, buf = 0; c0 < cnt; c0 += CH, buf ^= 1) {
    const int n = min(CH, cnt - c0);
    float* v = s_v + buf * (CH * kScanCols);
    float* sc = s_s + buf * (CH * 2);
#pragma unroll
    for (int i = 0; i < NVR; ++i)
      if (tid + NT * i < CH * kScanCols) v[tid + NT * i] = r_v[i];
    if (tid < CH) {
      if constexpr (SCALAR) sc[2 * tid] = r_s[0];
      if constexpr (MODE == 2) sc[2 * tid + 1] = r_s[1];
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();   // this chunk is there; the chunk before has been walked and handed out
    if (c0 + CH < cnt) {
      stage(c0 + CH, buf ^ 1);
      fetch(c0 + CH);
    }
    const float* x = s_x + buf * (CH * NV * DK) + d0;
    auto walk = [&](int t, auto group) {   // `group` tokens from t on: their operands load, and their parts leave, side by side
      constexpr int U = decltype(group)::value, W = RS < 4 ? 1 : 2;   // pairs of rows per load
      float dot[U][4];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const float4 vf = *reinterpret_cast<const float4*>(v + (t + u) * kScanCols + c4);
        const uint64_t vj[4] = {pair2(vf.x, vf.x), pair2(vf.y, vf.y), pair2(vf.z, vf.z), pair2(vf.w, vf.w)};
        const uint64_t ds = SCALAR ? pair2(sc[2 * (t + u)], sc[2 * (t + u)]) : 0;
        const float* xt = x + (t + u) * (NV * DK);
        uint64_t acc[4];
#pragma unroll
        for (int i0 = 0; i0 < RS / 2; i0 += W) {
          uint64_t b[W], r[W], d[W];
          auto load = [&](uint64_t(&o)[W], const float* q) {
            if constexpr (W == 2) {
              const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(q);
              o[0] = w.x;
              o[1] = w.y;
            } else {
              o[0] = *reinterpret_cast<const unsigned long long*>(q);
            }
          };
          load(b, xt + 2 * i0);
          load(r, xt + DK + 2 * i0);
          if constexpr (!SCALAR) load(d, xt + 2 * DK + 2 * i0);
#pragma unroll
          for (int i = 0; i < W; ++i) {
            const uint64_t dd = SCALAR ? ds : d[i];
#pragma unroll
            for (int c = 0; c < 4; ++c) {
              const uint64_t old = S[i0 + i][c];
              const uint64_t sn = fma2(b[i], vj[c], MODE == 0 ? mul2(dd, old) : fma2(dd, old, old));
              S[i0 + i][c] = sn;
              const uint64_t w = MODE == 2 ? old : sn;
              acc[c] = i0 + i == 0 ? mul2(w, r[i]) : fma2(w, r[i], acc[c]);
            }
          }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float2 a = split2(acc[c]);
          dot[u][c] = a.x + a.y;
        }
      }
      // four columns over the warp's eight row slices (lane bits 2 … 4): halves of the columns change hands twice, then a sum
      const bool h4 = lane & 16, h3 = lane & 8;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        float k0 = h4 ? dot[u][2] : dot[u][0], k1 = h4 ? dot[u][3] : dot[u][1];
        k0 += __shfl_xor_sync(0xffffffffu, h4 ? dot[u][0] : dot[u][2], 16);
        k1 += __shfl_xor_sync(0xffffffffu, h4 ? dot[u][1] : dot[u][3], 16);
        float k = h3 ? k1 : k0;
        k += __shfl_xor_sync(0xffffffffu, h3 ? k0 : k1, 8);
        k += __shfl_xor_sync(0xffffffffu, k, 4);
        if (!(lane & 4)) s_part[((t + u) * NW + warp) * kScanCols + c4 + (h4 ? 2 : 0) + (h3 ? 1 : 0)] = k;
      }
    };
    constexpr int G = RS <= 4 ? 4 : RS <= 8 ? 2 : 1;
    int t = 0;
    for (; t + G <= n; t += G) walk(t, std::integral_constant<int, G>{});
    for (; t < n; ++t) walk(t, std::integral_constant<int, 1>{});
    __syncthreads();
    for (int e = tid; e < n * kScanCols; e += NT) {
      const int t = e / kScanCols, c = e % kScanCols, cj = blockIdx.z * kScanCols + c;
      const float* q = s_part + t * NW * kScanCols + c;
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < NW; ++w) o += q[w * kScanCols];
      if constexpr (MODE == 2) o = fmaf(sc[2 * t + 1], v[e], o);
      if (cj < dv) p.o[(int64_t)(r0 + c0 + t) * p.ld_o + (int64_t)hd * dv + cj] = o;
    }
  }
#pragma unroll
  for (int i = 0; i < RS / 2; ++i)
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const float2 a = split2(S[i][c]);
      if (held(2 * i, c)) st[(int64_t)(d0 + 2 * i) * dv + j0 + c] = a.x;
      if (held(2 * i + 1, c)) st[(int64_t)(d0 + 2 * i + 1) * dv + j0 + c] = a.y;
    }
}

template <int RS, int NT, int MODE, bool SCALAR>
int launch_scan_cols(const LinScan& p, cudaStream_t st) {
  constexpr int smem = ScanCols<RS, NT, SCALAR>::smem;
  static cudaError_t attr = cudaFuncSetAttribute(lin_scan_cols_kernel<RS, NT, MODE, SCALAR>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  B200_CUDA(attr);
  auto al = [](const float* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool wide = p.dk % 4 == 0 && p.ld % 4 == 0 && al(p.b) && al(p.r) && (SCALAR || al(p.d));
  const dim3 grid(p.n_seg, p.heads, (p.dv + kScanCols - 1) / kScanCols);
  B200_CUDA(launch_pdl(lin_scan_cols_kernel<RS, NT, MODE, SCALAR>, grid, dim3(NT), smem, st, stack_pdl(), p, wide));
  return B200_OK;
}
template <int RS, int NT>
int launch_scan_cols(const LinScan& p, cudaStream_t st) {
  if (p.read_old) return launch_scan_cols<RS, NT, 2, false>(p, st);
  if (p.d_minus_one) return launch_scan_cols<RS, NT, 1, false>(p, st);
  return p.d_scalar ? launch_scan_cols<RS, NT, 0, true>(p, st) : launch_scan_cols<RS, NT, 0, false>(p, st);
}

// ------------------------------------------------------------------------------------------- generalized delta rule
// One warp per (token, head): decay w = exp(−c·sigmoid(wl)), removal a = sigmoid(logit), unit key u = k / sqrt(Σk² + ε); the
// scan's rows [decay | a∘u | u | k | r | v] in fp32.
template <typename T>
__global__ void __launch_bounds__(128) delta_prep_kernel(const DeltaRun p) {
  pdl_trigger();
  pdl_wait();
  const int pair = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int H = p.a.heads, dk = p.a.dim, dv = p.a.vdim;
  if (pair >= p.scan.n_tok * H) return;
  const int t = pair / H, hd = pair % H;
  const T* row = static_cast<const T*>(p.proj) + (int64_t)t * p.ld_proj;
  const T* k = row + p.off_k + hd * dk;
  float ss = 0.f;
  for (int i = lane; i < dk; i += 32) {
    const float v = ldf<T>(k + i);
    ss += v * v;
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) + p.d.unit_eps);
  float* f = p.f + (int64_t)t * p.scan.ld;
  const int64_t n = (int64_t)H * dk;
  for (int i = lane; i < dk; i += 32) {
    const int c = hd * dk + i;
    const float kv = ldf<T>(k + i), u = kv * inv;
    f[c] = expf(-p.d.decay_scale * sigmoidf(p.wl[(int64_t)t * n + c]));
    f[n + c] = sigmoidf(ldf<T>(row + p.off_a + c)) * u;
    f[2 * n + c] = u;
    f[3 * n + c] = kv;
    f[4 * n + c] = ldf<T>(row + p.off_r + c);
  }
  for (int i = lane; i < dv; i += 32) f[5 * n + hd * dv + i] = ldf<T>(row + p.off_v + hd * dv + i);
}

// One warp per (token, head): o / rms(o) · head_norm · sigmoid(out gate)
template <typename T>
__global__ void __launch_bounds__(128) delta_out_kernel(const DeltaRun p) {
  pdl_trigger();
  pdl_wait();
  const int pair = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int H = p.a.heads, dv = p.a.vdim;
  if (pair >= p.scan.n_tok * H) return;
  const int t = pair / H, hd = pair % H;
  const float* o = p.scan.o + (int64_t)t * p.scan.ld_o + hd * dv;
  float ss = 0.f;
  for (int c = lane; c < dv; c += 32) ss += o[c] * o[c];
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
  const T* g = static_cast<const T*>(p.proj) + (int64_t)t * p.ld_proj + p.off_g + hd * dv;
  T* y = static_cast<T*>(p.mid) + (int64_t)t * p.ld_mid + hd * dv;
  for (int c = lane; c < dv; c += 32) y[c] = cvt<T>(o[c] * inv * p.d.head_norm[hd * dv + c] * sigmoidf(ldf<T>(g + c)));
}

// -------------------------------------------------------------------------------------------------------------- Mamba-2
// The rows of a sequence lie side by side in the step, in order: row t − j is position pos[t] − j of the same sequence
// exactly when it has the same slot and that position.  Inputs from before the step's first row come from the slot's
// state, which holds the last taps − 1 inputs, oldest first (zeros before position 0).
__device__ __forceinline__ bool same_seq(const int32_t* slot, const int32_t* pos, int t, int j) {
  return row_same_seq(slot, pos, t, j);
}

// One thread per (row, channel): convolution over the row's own input and the taps − 1 before it + bias + SiLU into the
// fp32 workspace.  The state is only READ here (mamba_out_kernel, a later launch, moves it on).  The threads past the
// channels serve one head each: dt = softplus(logit + bias) and the decay exp(−exp(A_log)·dt).
template <typename T>
__global__ void __launch_bounds__(128) mamba_conv_kernel(const MambaRun p) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, c = blockIdx.y * 128 + threadIdx.x;
  const int H = p.a.heads, inner = H * p.a.vdim, ch = inner + 2 * p.m.groups * p.m.state, taps = p.m.taps;
  if (c >= ch + H) return;
  float* f = p.f + (int64_t)t * p.scan.ld;
  if (c >= ch) {
    const int hd = c - ch;
    const float dt = softplusf(p.dt[(int64_t)t * p.ld_dt + hd] + p.m.dt_bias[hd]);
    f[ch + hd] = expf(-expf(p.m.A_log[hd]) * dt);
    f[ch + H + hd] = dt;
    return;
  }
  const int32_t *slot = p.scan.slot, *pos = p.scan.pos;
  const T* x = static_cast<const T*>(p.proj) + p.off_x + c;
  const float* cs = p.conv_state + (int64_t)slot[t] * p.scan.slot_stride;
  float acc = p.m.conv_b[c];
  int in_step = 0;   // rows of this sequence in front of row t, counted up to taps − 1
  while (in_step < taps - 1 && same_seq(slot, pos, t, in_step + 1)) ++in_step;
  for (int j = 0; j < taps; ++j) {   // j positions back; weight column taps − 1 − j
    float v = 0.f;
    if (j <= in_step) v = ldf<T>(x + (int64_t)(t - j) * p.ld_proj);
    else if (pos[t] - j >= 0) v = cs[(int64_t)(taps - 1 - (j - in_step)) * ch + c];   // j − in_step inputs before the step's first row
    acc = fmaf(p.m.conv_w[(int64_t)c * taps + taps - 1 - j], v, acc);
  }
  f[c] = siluf(acc);
}

// First CTA of a token: y = o + D·x, · silu(z), an RMS norm in norm_groups equal parts, · norm.  The other CTAs of a sequence's
// LAST row in the step move the slot's convolution state on: the last taps − 1 inputs, from the step's rows where it has that
// many, else from the old state shifted in place.
template <typename T>
__global__ void __launch_bounds__(256) mamba_out_kernel(const MambaRun p) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const int t = blockIdx.x, tid = threadIdx.x;
  const int H = p.a.heads, dv = p.a.vdim, inner = H * dv, part = inner / p.m.norm_groups;
  if (blockIdx.y > 0) {   // the CTAs behind the first move the state on, 256 channels each
    const int32_t *slot = p.scan.slot, *pos = p.scan.pos;
    const int taps = p.m.taps, ch = inner + 2 * p.m.groups * p.m.state;
    const bool last = t + 1 >= p.scan.n_tok || slot[t + 1] != slot[t] || pos[t + 1] != pos[t] + 1;
    if (last && taps > 1) {
      int in_step = 0;
      while (in_step < taps - 1 && same_seq(slot, pos, t, in_step + 1)) ++in_step;
      float* cs = p.conv_state + (int64_t)slot[t] * p.scan.slot_stride;
      const T* x = static_cast<const T*>(p.proj) + p.off_x;
      for (int c = (blockIdx.y - 1) * 256 + tid; c < ch; c += 256 * (gridDim.y - 1)) {
        // new entry i = the input taps − 2 − i positions back from row t: a step row, or the old entry i + 1 + in_step — always
        // further along than anything written so far, so the shift runs in place
        for (int i = 0; i < taps - 1; ++i) {
          const int j = taps - 2 - i;
          float v = 0.f;
          if (j <= in_step) v = ldf<T>(x + (int64_t)(t - j) * p.ld_proj + c);
          else if (pos[t] - j >= 0) v = cs[(int64_t)(i + 1 + in_step) * ch + c];
          cs[(int64_t)i * ch + c] = v;
        }
      }
    }
    return;
  }
  const float* o = p.scan.o + (int64_t)t * p.scan.ld_o;
  const float* x = p.f + (int64_t)t * p.scan.ld;
  const T* z = static_cast<const T*>(p.proj) + (int64_t)t * p.ld_proj + p.off_z;
  T* y = static_cast<T*>(p.mid) + (int64_t)t * p.ld_mid;
  for (int g = 0; g < p.m.norm_groups; ++g) {
    float ss = 0.f;
    for (int i = g * part + tid; i < (g + 1) * part; i += 256) {
      const float v = (o[i] + p.m.D[i / dv] * x[i]) * siluf(ldf<T>(z + i));
      ss += v * v;
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)part + p.eps);
    for (int i = g * part + tid; i < (g + 1) * part; i += 256) {
      const float v = (o[i] + p.m.D[i / dv] * x[i]) * siluf(ldf<T>(z + i));
      y[i] = cvt<T>(v * inv * p.m.norm[i]);
    }
  }
}

// ------------------------------------------------------------------------------------------------- gated delta rule
// Channel c of the convolved q | k | v → its column in the projection rows
__device__ __forceinline__ int gdelta_col(const GatedDeltaRun& p, int c, int nqk) {
  return c < nqk ? p.off_q + c : c < 2 * nqk ? p.off_k + (c - nqk) : p.off_v + (c - 2 * nqk);
}

// One CTA per (token, query / key head g): the channels of q head g, k head g and the value heads that read them.  First the
// short causal convolution of every such channel over the row's own input and the taps − 1 before it (rows of the same
// sequence in this step, else the slot's state; zeros before position 0), then SiLU, into shared memory.  Then q and k
// become unit vectors (q also times dim^(−1/2)), and one warp per value head: its write strength beta = sigmoid(·), its decay
// g = exp(−exp(A_log)·softplus(· + dt_bias)).  The scan's fp32 rows:
//   [g: H | beta·g·k (the removal's weight vector): H·dk | k: G·dk | q: G·dk | v: H·dv | beta: H]
// The state is only READ here (gdelta_out_kernel, a later launch, moves it on).
template <typename T>
__global__ void __launch_bounds__(256) gdelta_prep_kernel(const GatedDeltaRun p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];   // [dk: q | dk: k | per·dv: v] convolved channels of this group
  const int t = blockIdx.x, g = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = p.a.heads, G = p.a.kv_heads, dk = p.a.dim, dv = p.a.vdim, taps = p.d.taps, per = H / G;
  const int nqk = G * dk, ch = 2 * nqk + H * dv, mine = 2 * dk + per * dv;
  const int32_t *slot = p.scan.slot, *pos = p.scan.pos;
  const T* proj = static_cast<const T*>(p.proj);
  const float* cs = p.conv_state + (int64_t)slot[t] * p.scan.slot_stride;
  int in_step = 0;   // rows of this sequence in front of row t, counted up to taps − 1
  while (in_step < taps - 1 && same_seq(slot, pos, t, in_step + 1)) ++in_step;
  for (int e = tid; e < mine; e += 256) {
    // the group's e-th channel → its place c among the q | k | v channels
    const int c = e < dk ? g * dk + e : e < 2 * dk ? nqk + g * dk + (e - dk) : 2 * nqk + g * per * dv + (e - 2 * dk);
    const int col = gdelta_col(p, c, nqk);
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {   // j positions back; weight column taps − 1 − j
      float v = 0.f;
      if (j <= in_step) v = ldf<T>(proj + (int64_t)(t - j) * p.ld_proj + col);
      else if (pos[t] - j >= 0) v = cs[(int64_t)(taps - 1 - (j - in_step)) * ch + c];
      acc = fmaf(p.d.conv_w[(int64_t)c * taps + taps - 1 - j], v, acc);
    }
    sm[e] = siluf(acc);
  }
  __syncthreads();
  float* f = p.f + (int64_t)t * p.scan.ld;
  float* f_g = f;
  float* f_p = f + H;
  float* f_k = f_p + (int64_t)H * dk;
  float* f_q = f_k + nqk;
  float* f_v = f_q + nqk;
  float* f_beta = f_v + (int64_t)H * dv;
  if (warp < 2) {   // warp 0: the unit query, warp 1: the unit key (kept in shared memory for the value heads)
    float* x = sm + warp * dk;
    float ss = 0.f;
    for (int i = lane; i < dk; i += 32) ss += x[i] * x[i];
    float inv = 1.f / sqrtf(warp_sum(ss) + p.d.unit_eps);
    if (warp == 0) inv *= rsqrtf((float)dk);
    float* dst = (warp == 0 ? f_q : f_k) + (int64_t)g * dk;
    for (int i = lane; i < dk; i += 32) {
      const float u = x[i] * inv;
      x[i] = u;
      dst[i] = u;
    }
  }
  __syncthreads();
  const T* row = proj + (int64_t)t * p.ld_proj;
  const float* k = sm + dk;
  for (int u = warp; u < per; u += 8) {
    const int hd = g * per + u;
    const float beta = sigmoidf(ldf<T>(row + p.off_b + hd));
    const float dec = expf(-expf(p.d.A_log[hd]) * softplusf(ldf<T>(row + p.off_a + hd) + p.d.dt_bias[hd]));
    if (lane == 0) {
      f_g[hd] = dec;
      f_beta[hd] = beta;
    }
    for (int i = lane; i < dk; i += 32) f_p[(int64_t)hd * dk + i] = beta * dec * k[i];
    for (int i = lane; i < dv; i += 32) f_v[(int64_t)hd * dv + i] = sm[2 * dk + u * dv + i];
  }
}

// First CTA of a token: one warp per head, o / rms(o) · head_norm (shared by the heads) · silu(out gate).  The other CTAs of a
// sequence's LAST row in the step move the slot's convolution state on: the last taps − 1 inputs, from the step's rows where
// it has that many, else from the old state shifted in place.
template <typename T>
__global__ void __launch_bounds__(256) gdelta_out_kernel(const GatedDeltaRun p) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = p.a.heads, G = p.a.kv_heads, dk = p.a.dim, dv = p.a.vdim;
  if (blockIdx.y > 0) {
    const int32_t *slot = p.scan.slot, *pos = p.scan.pos;
    const int taps = p.d.taps, nqk = G * dk, ch = 2 * nqk + H * dv;
    const bool last = t + 1 >= p.scan.n_tok || slot[t + 1] != slot[t] || pos[t + 1] != pos[t] + 1;
    if (last && taps > 1) {
      int in_step = 0;
      while (in_step < taps - 1 && same_seq(slot, pos, t, in_step + 1)) ++in_step;
      float* cs = p.conv_state + (int64_t)slot[t] * p.scan.slot_stride;
      const T* proj = static_cast<const T*>(p.proj);
      for (int c = (blockIdx.y - 1) * 256 + tid; c < ch; c += 256 * (gridDim.y - 1)) {
        const int col = gdelta_col(p, c, nqk);
        // new entry i = the input taps − 2 − i positions back from row t: a step row, or the old entry i + 1 + in_step — always
        // further along than anything written so far, so the shift runs in place
        for (int i = 0; i < taps - 1; ++i) {
          const int j = taps - 2 - i;
          float v = 0.f;
          if (j <= in_step) v = ldf<T>(proj + (int64_t)(t - j) * p.ld_proj + col);
          else if (pos[t] - j >= 0) v = cs[(int64_t)(i + 1 + in_step) * ch + c];
          cs[(int64_t)i * ch + c] = v;
        }
      }
    }
    return;
  }
  const T* g = static_cast<const T*>(p.proj) + (int64_t)t * p.ld_proj + p.off_g;
  T* y = static_cast<T*>(p.mid) + (int64_t)t * p.ld_mid;
  for (int hd = warp; hd < H; hd += 8) {
    const float* o = p.scan.o + (int64_t)t * p.scan.ld_o + hd * dv;
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) ss += o[c] * o[c];
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
    for (int c = lane; c < dv; c += 32) y[hd * dv + c] = cvt<T>(o[c] * inv * p.d.head_norm[c] * siluf(ldf<T>(g + hd * dv + c)));
  }
}

// --------------------------------------------------------------------------------------------------------- time mixing
// One warp per (token, head): decay exp(−exp(wl)) (minus one), the bonus Σ r·u·k; the scan's fp32 rows
// [decay − 1 | k | r | v | bonus].
template <typename T>
__global__ void __launch_bounds__(128) wkv_prep_kernel(const WkvRun p) {
  pdl_trigger();
  pdl_wait();
  const int pair = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int H = p.d.heads, dk = p.d.dim;
  if (pair >= p.scan.n_tok * H) return;
  const int t = pair / H, hd = pair % H;
  const int64_t n = (int64_t)H * dk, seg = (int64_t)p.scan.n_tok * n;
  const T* r = static_cast<const T*>(p.p4) + (int64_t)t * n;
  float* f = p.f + (int64_t)t * p.scan.ld;
  float b = 0.f;
  for (int i = lane; i < dk; i += 32) {
    const int c = hd * dk + i;
    const float rv = ldf<T>(r + c), kv = ldf<T>(r + seg + c);
    f[c] = expm1f(-expf(p.wl[(int64_t)t * n + c]));
    f[n + c] = kv;
    f[2 * n + c] = rv;
    f[3 * n + c] = ldf<T>(r + 2 * seg + c);
    b = fmaf(rv * p.d.u[c], kv, b);
  }
  b = warp_sum(b);
  if (lane == 0) f[4 * n + hd] = b;
}

// One warp per (token, head): o / rms(o) · norm · silu(gate) · scale; the last head's warp also clears the padding columns.
template <typename T>
__global__ void __launch_bounds__(128) wkv_out_kernel(const WkvRun p) {
  pdl_trigger();
  pdl_wait();
  const int pair = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int H = p.d.heads, dv = p.d.dim;
  if (pair >= p.scan.n_tok * H) return;
  const int t = pair / H, hd = pair % H;
  const int64_t n = (int64_t)H * dv;
  const float* o = p.scan.o + (int64_t)t * p.scan.ld_o + hd * dv;
  float ss = 0.f;
  for (int c = lane; c < dv; c += 32) ss += o[c] * o[c];
  const float inv = p.scale / sqrtf(warp_sum(ss) / (float)dv + p.eps);
  const T* g = static_cast<const T*>(p.p4) + ((int64_t)3 * p.scan.n_tok + t) * n + hd * dv;
  T* y = static_cast<T*>(p.mid) + (int64_t)t * p.ld_mid + hd * dv;
  for (int c = lane; c < dv; c += 32) y[c] = cvt<T>(o[c] * inv * p.d.norm[hd * dv + c] * siluf(ldf<T>(g + c)));
  if (hd == H - 1)
    for (int c = (int)n + lane; c < p.n_pad; c += 32) static_cast<T*>(p.mid)[(int64_t)t * p.ld_mid + c] = cvt<T>(0.f);
}

// ------------------------------------------------------------------------------------------------- gated linear attention
// log sigmoid(z)
__device__ __forceinline__ float log_sigmoidf(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// Prompts: kGlaStrip tokens × 256 columns per CTA.  A column is one of the heads·dim key channels (its decay minus one, from the
// strip's bottleneck rows in shared memory and its row of a2, and its key and query entries) or one of the heads·vdim value
// channels.  The scan's fp32 rows are [decay − 1 | k | q | v].
constexpr int kGlaStrip = 8;
template <typename T>
__global__ void __launch_bounds__(256) gla_prep_kernel(const GlaRun p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];   // [kGlaStrip][rank]
  const int t0 = blockIdx.x * kGlaStrip, n = min(kGlaStrip, p.scan.n_tok - t0), tid = threadIdx.x;
  const int H = p.a.heads, nk = H * p.a.dim, nv = H * p.a.vdim, rk = p.d.rank, ldw = (rk + 7) / 8 * 8;
  const int c = blockIdx.y * 256 + tid;
  const T* row = static_cast<const T*>(p.proj) + (int64_t)t0 * p.ld_proj;
  float* f = p.f + (int64_t)t0 * p.scan.ld;
  if (blockIdx.y * 256 < nk) {   // the same for the whole CTA
    for (int e = tid; e < kGlaStrip * rk; e += 256) sm[e] = e / rk < n ? ldf<T>(row + (int64_t)(e / rk) * p.ld_proj + p.off_a + e % rk) : 0.f;
    __syncthreads();
  }
  if (c < nk) {
    const float scale = 1.f / sqrtf((float)p.a.dim), inv_tau = 1.f / p.d.tau, b = p.d.a2_b[c];
    const T* w = static_cast<const T*>(p.d.a2) + (int64_t)c * ldw;
    float z[kGlaStrip];
#pragma unroll
    for (int u = 0; u < kGlaStrip; ++u) z[u] = b;
#pragma unroll 4
    for (int r = 0; r < rk; ++r) {
      const float wr = ldf<T>(w + r);
#pragma unroll
      for (int u = 0; u < kGlaStrip; ++u) z[u] = fmaf(wr, sm[u * rk + r], z[u]);
    }
#pragma unroll
    for (int u = 0; u < kGlaStrip; ++u) {
      if (u >= n) break;
      const T* x = row + (int64_t)u * p.ld_proj;
      float* o = f + (int64_t)u * p.scan.ld;
      o[c] = expm1f(log_sigmoidf(z[u]) * inv_tau);
      o[nk + c] = ldf<T>(x + p.off_k + c);
      o[2 * nk + c] = ldf<T>(x + p.off_q + c) * scale;
    }
  } else if (c >= (nk + 255) / 256 * 256) {
    const int cv = c - (nk + 255) / 256 * 256;
    if (cv < nv)
      for (int u = 0; u < n; ++u) f[(int64_t)u * p.scan.ld + 3 * nk + cv] = ldf<T>(row + (int64_t)u * p.ld_proj + p.off_v + cv);
  }
}

// One warp per (token, head): o / rms(o) · head_norm (shared by the heads) · silu(out gate).
template <typename T>
__global__ void __launch_bounds__(256) gla_out_kernel(const GlaRun p) {
  pdl_trigger();
  pdl_wait();
  const int64_t pair = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31, H = p.a.heads, dv = p.a.vdim;
  if (pair >= (int64_t)p.scan.n_tok * H) return;
  const int t = (int)(pair / H), hd = (int)(pair % H);
  const float* o = p.scan.o + (int64_t)t * p.scan.ld_o + hd * dv;
  float ss = 0.f;
  for (int c = lane; c < dv; c += 32) ss += o[c] * o[c];
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
  const T* g = static_cast<const T*>(p.proj) + (int64_t)t * p.ld_proj + p.off_g + hd * dv;
  T* y = static_cast<T*>(p.mid) + (int64_t)t * p.ld_mid + hd * dv;
  for (int c = lane; c < dv; c += 32) y[c] = cvt<T>(o[c] * inv * p.d.head_norm[c] * siluf(ldf<T>(g + c)));
}

// Steps in which every row is its sequence's only new one: the whole mixer between its two products in one launch.  One CTA per
// (row, head).  The state's entries a thread owns — one column, every `slices`-th … of kGlaRows rows — are requested ahead of
// the dependency wait (an earlier step left them there, and the row's slot and position come from the step's first kernel);
// behind it decays, keys, queries and values go to shared memory, the state moves on in registers and back to memory, the
// slices' sums of a column meet in shared memory, and the head's norm and gate follow.
constexpr int kGlaThreads = 512;
constexpr int kGlaRows = 32;
template <typename T>
__global__ void __launch_bounds__(kGlaThreads) gla_step_kernel(const GlaRun p) {
  pdl_trigger();
  extern __shared__ float sm[];
  __shared__ float red[kGlaThreads / 32];
  const int t = blockIdx.x, hd = blockIdx.y, tid = threadIdx.x;
  const int H = p.a.heads, dk = p.a.dim, dv = p.a.vdim, rk = p.d.rank, ldw = (rk + 7) / 8 * 8;
  const int cw = min(kGlaThreads, (dv + 31) / 32 * 32), slices = kGlaThreads / cw;   // columns side by side; row slices
  const int per = (dk + slices - 1) / slices;
  float* s_d = sm;               // [dk] decay − 1
  float* s_k = s_d + dk;         // [dk]
  float* s_q = s_k + dk;         // [dk]
  float* s_u = s_q + dk;         // [rk]
  float* s_o = s_u + rk;         // [dv]
  float* s_p = s_o + dv;         // [slices][cw]
  const int slice = tid / cw, col = tid % cw;
  float* st = p.scan.state + (int64_t)p.scan.slot[t] * p.scan.slot_stride + (int64_t)hd * dk * dv;
  const bool fresh = p.scan.pos[t] == 0;
  const int d0 = slice * per, d1 = slice < slices ? min(dk, d0 + per) : d0;
  float S[kGlaRows];
  auto fetch = [&](int j, int d) {
#pragma unroll
    for (int i = 0; i < kGlaRows; ++i) S[i] = d + i < d1 && j < dv && !fresh ? st[(int64_t)(d + i) * dv + j] : 0.f;
  };
  fetch(col, d0);
  pdl_wait();
  const T* row = static_cast<const T*>(p.proj) + (int64_t)t * p.ld_proj;
  for (int i = tid; i < rk; i += kGlaThreads) s_u[i] = ldf<T>(row + p.off_a + i);
  for (int i = tid; i < dk; i += kGlaThreads) {
    s_k[i] = ldf<T>(row + p.off_k + hd * dk + i);
    s_q[i] = ldf<T>(row + p.off_q + hd * dk + i) * (1.f / sqrtf((float)dk));
  }
  __syncthreads();
  for (int i = tid; i < dk; i += kGlaThreads) {
    const T* w = static_cast<const T*>(p.d.a2) + (int64_t)(hd * dk + i) * ldw;
    float z = p.d.a2_b[hd * dk + i];
#pragma unroll 8
    for (int r = 0; r < rk; ++r) z = fmaf(ldf<T>(w + r), s_u[r], z);
    s_d[i] = expm1f(log_sigmoidf(z) * (1.f / p.d.tau));
  }
  __syncthreads();
  float ss = 0.f;
  for (int j0 = 0; j0 < dv; j0 += cw) {
    const int j = j0 + col;
    const float v = j < dv ? ldf<T>(row + p.off_v + hd * dv + j) : 0.f;
    float acc = 0.f;
    for (int d = d0; d < d1; d += kGlaRows) {
      if (j0 > 0 || d > d0) fetch(j, d);
#pragma unroll
      for (int i = 0; i < kGlaRows; ++i) {
        if (d + i < d1 && j < dv) {
          const float sn = fmaf(s_k[d + i], v, fmaf(s_d[d + i], S[i], S[i]));
          st[(int64_t)(d + i) * dv + j] = sn;
          acc = fmaf(sn, s_q[d + i], acc);
        }
      }
    }
    if (slice < slices) s_p[tid] = acc;
    __syncthreads();
    if (tid < cw && j < dv) {
      float o = 0.f;
      for (int s = 0; s < slices; ++s) o += s_p[s * cw + tid];
      s_o[j] = o;
      ss += o * o;
    }
    __syncthreads();
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)dv + p.eps);
  T* y = static_cast<T*>(p.mid) + (int64_t)t * p.ld_mid + hd * dv;
  for (int c = tid; c < dv; c += kGlaThreads) y[c] = cvt<T>(s_o[c] * inv * p.d.head_norm[c] * siluf(ldf<T>(row + p.off_g + hd * dv + c)));
}

// ------------------------------------------------------------------------------------------------------ selective scan
// One thread per (row, channel): convolution over the row's own input and the taps − 1 before it, bias, SiLU.
template <typename T>
__global__ void __launch_bounds__(128) mamba1_conv_kernel(const Mamba1Run p) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, c = blockIdx.y * 128 + threadIdx.x, inner = p.d.inner, taps = p.d.taps;
  if (c >= inner) return;
  const T* x = static_cast<const T*>(p.proj) + p.off_x + c;
  float* cs = p.conv_state + (int64_t)p.slot[t] * p.slot_stride;
  const int front = rows_in_front(p.slot, p.pos, t, taps - 1), ps = p.pos[t];
  auto back = [&](int j) {
    if (j <= front) return ldf<T>(x + (int64_t)(t - j) * p.ld_proj);
    return ps - j >= 0 ? cs[(int64_t)(taps - 1 - (j - front)) * inner + c] : 0.f;
  };
  float acc = p.d.conv_b[c];
  for (int j = 0; j < taps; ++j) acc = fmaf(p.d.conv_w[(int64_t)(taps - 1 - j) * inner + c], back(j), acc);
  static_cast<T*>(p.xc)[(int64_t)t * inner + c] = cvt<T>(siluf(acc));
  if (p.advance)
    for (int e = 0; e < taps - 1; ++e) {   // entry e: the row taps − 2 − e positions back, further along than what is written
      const float v = back(taps - 2 - e);
      cs[(int64_t)e * inner + c] = v;
    }
}

// Prompts: kM1Strip rows and two neighbouring channels per thread; while a sequence goes on, the window slides through registers.
constexpr int kM1Strip = 16;
__device__ __forceinline__ float2 ld2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ld2(const __nv_bfloat16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void st2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void st2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) mamba1_conv_strip_kernel(const Mamba1Run p) {
  pdl_trigger();
  const int t0 = blockIdx.x * kM1Strip, c = (blockIdx.y * 128 + threadIdx.x) * 2, inner = p.d.inner;
  const bool mine = c < inner;
  float2 w[TAPS], win[TAPS], bias = make_float2(0.f, 0.f);
  if (mine) {
    bias = ld2(p.d.conv_b + c);
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = ld2(p.d.conv_w + (int64_t)j * inner + c);
  }
  pdl_wait();
  if (!mine) return;
  const T* x = static_cast<const T*>(p.proj) + p.off_x + c;
  const int t1 = min(t0 + kM1Strip, p.n_tok);
  const bool one = rows_one_seq(p.slot, p.pos, t0, t1);
#pragma unroll 4
  for (int t = t0; t < t1; ++t) {
    if (t == t0 || (!one && !row_same_seq(p.slot, p.pos, t, 1))) {
      const int front = rows_in_front(p.slot, p.pos, t, TAPS - 1), ps = p.pos[t];
      const float* cs = p.conv_state + (int64_t)p.slot[t] * p.slot_stride + c;
#pragma unroll
      for (int j = 1; j < TAPS; ++j)
        win[j] = j <= front ? ld2(x + (int64_t)(t - j) * p.ld_proj) : ps - j >= 0 ? ld2(cs + (int64_t)(TAPS - 1 - (j - front)) * inner) : make_float2(0.f, 0.f);
    } else {
#pragma unroll
      for (int j = TAPS - 1; j > 0; --j) win[j] = win[j - 1];
    }
    win[0] = ld2(x + (int64_t)t * p.ld_proj);
    float2 a = bias;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      a.x = fmaf(w[TAPS - 1 - j].x, win[j].x, a.x);
      a.y = fmaf(w[TAPS - 1 - j].y, win[j].y, a.y);
    }
    st2(static_cast<T*>(p.xc) + (int64_t)t * inner + c, siluf(a.x), siluf(a.y));
  }
}

// One warp per (row, channel): dt logit = Σ_r w_dt[c][r]·T(dt_r) + dt_b
template <typename T>
__global__ void __launch_bounds__(256) mamba1_dt_kernel(const Mamba1Run p) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, t = blockIdx.y;
  if (c >= p.d.inner) return;
  const int rk8 = (p.d.dt_rank + 7) / 8 * 8;
  const T* w = static_cast<const T*>(p.d.w_dt) + (int64_t)c * rk8;
  const float* x = p.xd + (int64_t)t * p.ld_xd;
  float a = 0.f;
  for (int i = lane; i < p.d.dt_rank; i += 32) a = fmaf(ldf<T>(w + i), x[i], a);
  a = warp_sum(a);
  if (lane == 0) p.dt[(int64_t)t * p.d.inner + c] = a + p.d.dt_b[c];
}

// 2^x and the two gates by the hardware's approximate exponential, logarithm and reciprocal (relative errors of about 2^-22; bf16
// engines), or as CUDA's functions (fp32 engines).
__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <typename T> __device__ __forceinline__ float gate_softplus(float z) { return softplusf(z); }
template <> __device__ __forceinline__ float gate_softplus<__nv_bfloat16>(float z) {
  const float e = ex2_fast(-fabsf(z) * 1.4426950408889634f);   // log(1 + e): its series where the sum would lose e's digits
  return fmaxf(z, 0.f) + (e < 0.01f ? e * (1.f - e * (0.5f - 0.33333333f * e)) : __logf(1.f + e));
}
template <typename T> __device__ __forceinline__ float gate_silu(float z) { return siluf(z); }
template <> __device__ __forceinline__ float gate_silu<__nv_bfloat16>(float z) {
  return __fdividef(z, 1.f + ex2_fast(fminf(-z * 1.4426950408889634f, 80.f)));
}

// LPC lanes share a channel, NPT state entries each; 256 threads = 256 / LPC channels per CTA.  The CTA walks its sequence CH
// tokens at a time: the chunk's B and C rows (fp32) and its channels' step sizes, inputs and gates sit in shared memory,
// while the next chunk's values are already on their way into registers.  The state is in registers for the whole walk; a
// token costs a thread NPT exponentials and 3·NPT multiply-adds, and the lanes' partial sums of four tokens meet side by
// side, off the state's chain, each pair of lanes keeping half of the tokens.  The decay is 2^(dt·A·log2 e); fp32 engines take
// exp(dt·A) − 1 instead, so that thousands of decays close to one do not add up a rounding of their own.  Entries past the
// state's size hold zeros (decay 1, B = C = 0).  A chunk's outputs leave together.
template <typename T, int LPC, int NPT>
__global__ void __launch_bounds__(256) mamba1_scan_kernel(const Mamba1Run p) {
  pdl_trigger();
  pdl_wait();
  constexpr int NS = LPC * NPT, CPB = 256 / LPC;
  constexpr int CH = NS <= 32 ? 32 : NS <= 64 ? 16 : 8;         // tokens per chunk
  constexpr int NBC = CH * 2 * NS / 256;                        // staged B | C entries per thread
  constexpr int NX = (CH * CPB + 255) / 256;                    // staged (token, channel) triples per thread
  static_assert(LPC >= 4 && CH * 2 * NS % 256 == 0, "mamba1 scan tiling");
  __shared__ float s_b[CH][NS], s_c[CH][NS];
  __shared__ float2 s_d[CH][CPB];                               // step size, step size · input
  __shared__ float2 s_o[CH][CPB];                               // D · input, gate
  __shared__ float s_y[CH][CPB];
  const int seg = blockIdx.x, tid = threadIdx.x, ch = tid / LPC, ln = tid % LPC;
  const int c0 = blockIdx.y * CPB, c = c0 + ch, inner = p.d.inner, N = p.d.state;
  const int r0 = p.seg_row0 != nullptr ? p.seg_row0[seg] : seg;
  const int cnt = p.seg_count != nullptr ? p.seg_count[seg] : 1;
  float* st = p.state + (int64_t)p.slot[r0] * p.slot_stride + (int64_t)c * N;
  const bool fresh = p.pos[r0] == 0, live = c < inner;
  float S[NPT], A[NPT];
#pragma unroll
  for (int i = 0; i < NPT; ++i) {   // lane ln holds entries ln·NPT …: consecutive B / C entries per thread
    const int n = ln * NPT + i;
    S[i] = live && n < N && !fresh ? st[n] : 0.f;
    A[i] = live && n < N ? -expf(p.d.A_log[(int64_t)c * N + n]) * (sizeof(T) == 4 ? 1.f : 1.4426950408889634f) : 0.f;
  }
  const int off_b = (p.d.dt_rank + 7) / 8 * 8;
  float r_bc[NBC], r_dt[NX];
  T r_x[NX], r_z[NX];   // as they lie in memory: widening them here would wait for the loads
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < NBC; ++i) {
      const int e = tid + 256 * i, t = e / (2 * NS), w = (e / NS) & 1, n = e % NS;
      r_bc[i] = t0 + t < cnt && n < N ? p.xd[(int64_t)(r0 + t0 + t) * p.ld_xd + off_b + w * N + n] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NX; ++i) {
      const int e = tid + 256 * i, t = e / CPB, cc = c0 + e % CPB;
      r_dt[i] = -INFINITY;   // rows past the end: step size softplus(−inf) = 0, the state stays
      r_x[i] = r_z[i] = cvt<T>(0.f);
      if (e < CH * CPB && t0 + t < cnt && cc < inner) {
        const int64_t row = r0 + t0 + t;
        r_dt[i] = p.dt[row * inner + cc];
        r_x[i] = static_cast<const T*>(p.xc)[row * inner + cc];
        r_z[i] = static_cast<const T*>(p.proj)[row * p.ld_proj + p.off_z + cc];
      }
    }
  };
  auto flush = [&](int t0) {   // the outputs of the chunk that starts at t0
#pragma unroll
    for (int i = 0; i < NX; ++i) {
      const int e = tid + 256 * i, t = e / CPB, cc = e % CPB;
      if (e < CH * CPB && t0 + t < cnt && c0 + cc < inner) {
        const float2 o = s_o[t][cc];
        static_cast<T*>(p.mid)[(int64_t)(r0 + t0 + t) * p.ld_mid + c0 + cc] = cvt<T>((s_y[t][cc] + o.x) * o.y);
      }
    }
  };
  float D[NX];
#pragma unroll
  for (int i = 0; i < NX; ++i) {
    const int cc = c0 + (tid + 256 * i) % CPB;
    D[i] = cc < inner ? p.d.D[cc] : 0.f;
  }
  const bool hi1 = (ln & (LPC / 2)) != 0, hi2 = (ln & (LPC / 4)) != 0, owner = (ln & (LPC / 4 - 1)) == 0;
  const int own = (hi1 ? 2 : 0) + (hi2 ? 1 : 0);   // which of four tokens this lane ends up with
  fetch(0);
  for (int t0 = 0; t0 < cnt; t0 += CH) {
    __syncthreads();
    if (t0 > 0) flush(t0 - CH);
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NBC; ++i) {
      const int e = tid + 256 * i, t = e / (2 * NS), w = (e / NS) & 1, n = e % NS;
      (w ? s_c : s_b)[t][n] = r_bc[i];
    }
#pragma unroll
    for (int i = 0; i < NX; ++i) {
      const int e = tid + 256 * i;
      if (e < CH * CPB) {
        const float dt = r_dt[i] == -INFINITY ? 0.f : gate_softplus<T>(r_dt[i]), x = ldf<T>(&r_x[i]);
        (&s_d[0][0])[e] = make_float2(dt, dt * x);
        (&s_o[0][0])[e] = make_float2(D[i] * x, gate_silu<T>(ldf<T>(&r_z[i])));
      }
    }
    __syncthreads();
    if (t0 + CH < cnt) fetch(t0 + CH);
    const int n4 = min(CH, (cnt - t0 + 3) / 4 * 4);
    for (int t4 = 0; t4 < n4; t4 += 4) {
      float y[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int t = t4 + u;
        const float2 d = s_d[t][ch];
        float a = 0.f;
#pragma unroll
        for (int i = 0; i < NPT; ++i) {
          const float b = s_b[t][ln * NPT + i];
          if constexpr (sizeof(T) == 4) S[i] += fmaf(expm1f(d.x * A[i]), S[i], d.y * b);
          else S[i] = fmaf(ex2_fast(d.x * A[i]), S[i], d.y * b);
          a = fmaf(S[i], s_c[t][ln * NPT + i], a);
        }
        y[u] = a;
      }
      float a0 = hi1 ? y[2] : y[0], a1 = hi1 ? y[3] : y[1];
      a0 += __shfl_xor_sync(0xffffffffu, hi1 ? y[0] : y[2], LPC / 2);
      a1 += __shfl_xor_sync(0xffffffffu, hi1 ? y[1] : y[3], LPC / 2);
      float a = hi2 ? a1 : a0;
      a += __shfl_xor_sync(0xffffffffu, hi2 ? a0 : a1, LPC / 4);
#pragma unroll
      for (int o = LPC / 8; o > 0; o >>= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
      if (owner) s_y[t4 + own][ch] = a;
    }
  }
  __syncthreads();
  flush((cnt - 1) / CH * CH);
  if (!live) return;
#pragma unroll
  for (int i = 0; i < NPT; ++i) {
    const int n = ln * NPT + i;
    if (n < N) st[n] = S[i];
  }
}

template <typename T>
__global__ void __launch_bounds__(256) stack_cast_rows_kernel(T* __restrict__ y, int64_t ld_y, const float* __restrict__ x, int64_t ld_x,
                                                              int n, int tanh_of, int64_t total) {
  pdl_trigger();
  pdl_wait();
  for (int64_t e = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (int64_t)gridDim.x * blockDim.x) {
    const float v = x[e / n * ld_x + e % n];
    y[e / n * ld_y + e % n] = cvt<T>(tanh_of ? tanhf(v) : v);
  }
}

// --------------------------------------------------------------------------------- post-norm + residual + operand copy
template <typename YT>
__global__ void __launch_bounds__(256) stack_rms_add_cast_kernel(float* __restrict__ x, const YT* __restrict__ y,
                                                                 const float* __restrict__ w, __nv_bfloat16* __restrict__ h,
                                                                 int dim, float eps, float mult) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const YT* yr = y + (int64_t)blockIdx.x * dim;
  float* xr = x + (int64_t)blockIdx.x * dim;
  float ss = 0.f;
  for (int i = threadIdx.x; i < dim; i += blockDim.x) ss += ldf<YT>(yr + i) * ldf<YT>(yr + i);
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)dim + eps);
  for (int i = threadIdx.x; i < dim; i += blockDim.x) {
    const float v = xr[i] + mult * (ldf<YT>(yr + i) * inv * w[i]);
    xr[i] = v;
    if (h != nullptr) h[(int64_t)blockIdx.x * dim + i] = __float2bfloat16_rn(v);
  }
}

// The same for a few rows that fit the CTA's registers (decode steps, where latency counts): y, w and x are requested
// together — one memory round trip before the reduction instead of three.  dim <= 16 · 256.
template <typename YT>
__global__ void __launch_bounds__(256) stack_rms_add_cast_small_kernel(float* __restrict__ x, const YT* __restrict__ y,
                                                                       const float* __restrict__ w, __nv_bfloat16* __restrict__ h,
                                                                       int dim, float eps, float mult) {
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const YT* yr = y + (int64_t)blockIdx.x * dim;
  float* xr = x + (int64_t)blockIdx.x * dim;
  float yv[16], wv[16], xv[16];
#pragma unroll
  for (int k = 0; k < 16; ++k) {
    const int i = threadIdx.x + k * 256;
    yv[k] = i < dim ? ldf<YT>(yr + i) : 0.f;
    wv[k] = i < dim ? w[i] : 0.f;
    xv[k] = i < dim ? xr[i] : 0.f;
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < 16; ++k) ss += yv[k] * yv[k];
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)dim + eps);
#pragma unroll
  for (int k = 0; k < 16; ++k) {
    const int i = threadIdx.x + k * 256;
    if (i < dim) {
      const float v = xv[k] + mult * (yv[k] * inv * wv[k]);
      xr[i] = v;
      if (h != nullptr) h[(int64_t)blockIdx.x * dim + i] = __float2bfloat16_rn(v);
    }
  }
}

}  // namespace

#define REC_DTYPE_CHECK(dtype) \
  B200_CHECK_ARG((dtype) == B200_BF16 || (dtype) == B200_F32, "stack op: unknown dtype %d", (int)(dtype))

int launch_attn_prep(const AttnPrep& p, int dtype, cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  B200_CHECK_ARG(p.proj && p.pos && p.n_tok > 0, "attention prep: null argument");
  B200_CHECK_ARG(p.d.rot_dims >= 0 && p.d.rot_dims % 2 == 0 && p.d.rot_dims <= p.a.dim && (p.d.rot_dims == 0 || p.d.rot_table),
                 "attention prep: rot_dims %d must be even, at most the head size %d, with a table", p.d.rot_dims, p.a.dim);
  B200_CHECK_ARG(!p.d.qk_norm || (p.d.q_norm && p.d.k_norm), "attention prep: null norm weight");
  B200_CHECK_ARG(p.d.v_mix >= 0 && p.d.v_mix <= 2 && (p.d.v_mix == 0 || p.vkeep) && (p.d.v_mix != 2 || p.d.mix_lambda),
                 "attention prep: value mix-in without its buffer or weight");
  if (dtype == B200_F32) B200_CUDA(launch_pdl(attn_prep_kernel<float>, dim3(p.n_tok), dim3(256), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(attn_prep_kernel<__nv_bfloat16>, dim3(p.n_tok), dim3(256), 0, st, stack_pdl(), p));
  return B200_OK;
}

int launch_lin_scan(const LinScan& p, cudaStream_t st) {
  B200_CHECK_ARG(p.d && p.b && p.r && p.v && p.state && p.slot && p.pos && p.o && p.n_seg > 0 && p.n_tok > 0,
                 "linear scan: null argument");
  B200_CHECK_ARG((p.p == nullptr) == (p.q == nullptr), "linear scan: the removal needs both of its vectors");
  B200_CHECK_ARG(p.heads > 0 && p.dk > 0 && p.dv > 0 && p.share > 0 && p.heads % p.share == 0, "linear scan: bad sizes");
  B200_CHECK_ARG(!p.d_scalar || (!p.read_old && !p.d_minus_one), "linear scan: a scalar decay is given as it is");
  B200_CHECK_ARG(!p.read_old || (p.p == nullptr && p.bonus && p.vscale == nullptr), "linear scan: reading the old state takes a bonus and no removal");
  B200_CHECK_ARG(!p.d_minus_one || p.p == nullptr, "linear scan: a decay minus one takes no removal");
  B200_CHECK_ARG(p.dk <= kScanMaxDim, "linear scan: more than %d key channels not built", kScanMaxDim);
  if (p.p == nullptr) {
    if (p.dk <= 64) return launch_scan_cols<2, 128>(p, st);
    if (p.dk <= 128) return launch_scan_cols<4, 128>(p, st);
    if (p.dk <= 256) return launch_scan_cols<4, 256>(p, st);
    return launch_scan_cols<8, 256>(p, st);
  }
  // two columns per warp where the value size fills them and the registers hold them: half the CTAs stage the same rows
  const int nc = (p.dv >= 32 && p.dk <= 256) ? 2 : 1;
  const dim3 grid(p.n_seg, p.heads, (p.dv + 8 * nc - 1) / (8 * nc));
#define B200_SCAN(DR)                                                                                           \
  do {                                                                                                          \
    if (nc == 2) B200_CUDA(launch_pdl(lin_scan_kernel<DR, 2>, grid, dim3(256), 0, st, stack_pdl(), p));          \
    else B200_CUDA(launch_pdl(lin_scan_kernel<DR, 1>, grid, dim3(256), 0, st, stack_pdl(), p));                  \
  } while (0)
  if (p.dk <= 32) B200_SCAN(1);
  else if (p.dk <= 64) B200_SCAN(2);
  else if (p.dk <= 128) B200_SCAN(4);
  else if (p.dk <= 256) B200_SCAN(8);
  else B200_SCAN(16);
#undef B200_SCAN
  return B200_OK;
}

int run_delta(const DeltaRun& p, int dtype, cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  B200_CHECK_ARG(p.proj && p.wl && p.f && p.scan.n_tok > 0, "delta rule: null argument");
  const int H = p.a.heads, dk = p.a.dim, dv = p.a.vdim;
  const dim3 grid((p.scan.n_tok * H + 3) / 4);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(delta_prep_kernel<float>, grid, dim3(128), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(delta_prep_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, stack_pdl(), p));
  LinScan s = p.scan;
  const int64_t n = (int64_t)H * dk;
  s.heads = H; s.dk = dk; s.dv = dv; s.share = 1; s.d_scalar = 0;
  s.d = p.f; s.p = p.f + n; s.q = p.f + 2 * n; s.b = p.f + 3 * n; s.r = p.f + 4 * n; s.v = p.f + 5 * n; s.vscale = nullptr;
  int rc = launch_lin_scan(s, st);
  if (rc != B200_OK || p.mid == nullptr) return rc;
  B200_CHECK_ARG(p.d.head_norm != nullptr, "delta rule: null head norm");
  if (dtype == B200_F32) B200_CUDA(launch_pdl(delta_out_kernel<float>, grid, dim3(128), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(delta_out_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, stack_pdl(), p));
  return B200_OK;
}

int run_gdelta(const GatedDeltaRun& p, int dtype, cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  B200_CHECK_ARG(p.proj && p.conv_state && p.f && p.mid && p.scan.n_tok > 0 && p.scan.n_seg > 0, "gated delta rule: null argument");
  const int H = p.a.heads, G = p.a.kv_heads, dk = p.a.dim, dv = p.a.vdim;
  B200_CHECK_ARG(H > 0 && G > 0 && H % G == 0 && dk > 0 && dv > 0, "gated delta rule: heads %d over %d query / key heads", H, G);
  B200_CHECK_ARG(p.d.taps >= 1 && p.d.taps <= kMambaMaxTaps, "gated delta rule: 1 … %d convolution taps", kMambaMaxTaps);
  B200_CHECK_ARG(p.d.conv_w && p.d.A_log && p.d.dt_bias && p.d.head_norm && p.d.unit_eps >= 0.f, "gated delta rule: null weight");
  const int nqk = G * dk, ch = 2 * nqk + H * dv;
  const size_t smem = (size_t)(2 * dk + (H / G) * dv) * 4;
  B200_CHECK_ARG(smem <= 200 * 1024, "gated delta rule: the channels of one query / key head and its value heads exceed one CTA's shared memory");
  if (smem > 48 * 1024) {
    static bool attr_done = false;
    if (!attr_done) {
      B200_CUDA(cudaFuncSetAttribute(gdelta_prep_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
      B200_CUDA(cudaFuncSetAttribute(gdelta_prep_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
      attr_done = true;
    }
  }
  const dim3 pg(p.scan.n_tok, G);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(gdelta_prep_kernel<float>, pg, dim3(256), smem, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(gdelta_prep_kernel<__nv_bfloat16>, pg, dim3(256), smem, st, stack_pdl(), p));
  LinScan s = p.scan;
  s.heads = H; s.dk = dk; s.dv = dv; s.share = H / G; s.d_scalar = 1; s.q_shared = 1;
  s.d = p.f; s.p = p.f + H; s.q = s.p + (int64_t)H * dk; s.b = s.q; s.r = s.q + nqk; s.v = s.r + nqk;
  s.vscale = s.v + (int64_t)H * dv;
  int rc = launch_lin_scan(s, st);
  if (rc != B200_OK) return rc;
  const dim3 og(p.scan.n_tok, p.d.taps > 1 ? 1 + std::min((ch + 255) / 256, 16) : 1);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(gdelta_out_kernel<float>, og, dim3(256), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(gdelta_out_kernel<__nv_bfloat16>, og, dim3(256), 0, st, stack_pdl(), p));
  return B200_OK;
}

int run_mamba(const MambaRun& p, int dtype, cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  B200_CHECK_ARG(p.proj && p.dt && p.conv_state && p.f && p.mid && p.scan.n_tok > 0 && p.scan.n_seg > 0, "mamba2: null argument");
  const b200_mamba_desc& m = p.m;
  const int H = p.a.heads, dv = p.a.vdim, N = m.state, inner = H * dv, ch = inner + 2 * m.groups * N;
  B200_CHECK_ARG(m.taps >= 1 && m.taps <= kMambaMaxTaps, "mamba2: 1 … %d convolution taps", kMambaMaxTaps);
  B200_CHECK_ARG(m.groups > 0 && H % m.groups == 0 && m.norm_groups > 0 && inner % m.norm_groups == 0 && N > 0,
                 "mamba2: heads %d, groups %d, norm_groups %d do not divide", H, m.groups, m.norm_groups);
  B200_CHECK_ARG(m.conv_w && m.conv_b && m.dt_bias && m.A_log && m.D && m.norm, "mamba2: null weight");
  const dim3 cg(p.scan.n_tok, (ch + H + 127) / 128);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(mamba_conv_kernel<float>, cg, dim3(128), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(mamba_conv_kernel<__nv_bfloat16>, cg, dim3(128), 0, st, stack_pdl(), p));
  LinScan s = p.scan;
  s.heads = H; s.dk = N; s.dv = dv; s.share = H / m.groups; s.d_scalar = 1;
  s.v = p.f; s.b = p.f + inner; s.r = p.f + inner + (int64_t)m.groups * N; s.d = p.f + ch; s.vscale = p.f + ch + H;
  s.p = s.q = nullptr;
  int rc = launch_lin_scan(s, st);
  if (rc != B200_OK) return rc;
  const dim3 og(p.scan.n_tok, m.taps > 1 ? 1 + std::min((ch + 255) / 256, 16) : 1);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(mamba_out_kernel<float>, og, dim3(256), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(mamba_out_kernel<__nv_bfloat16>, og, dim3(256), 0, st, stack_pdl(), p));
  return B200_OK;
}

int run_wkv(const WkvRun& p, int dtype, cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  const int H = p.d.heads, dk = p.d.dim;
  B200_CHECK_ARG(p.p4 && p.wl && p.f && p.mid && p.scan.n_tok > 0 && H > 0 && dk > 0, "time mixing: null argument");
  B200_CHECK_ARG(p.d.u && p.d.norm, "time mixing: null weight");
  const dim3 grid((unsigned)(((int64_t)p.scan.n_tok * H + 3) / 4));
  if (dtype == B200_F32) B200_CUDA(launch_pdl(wkv_prep_kernel<float>, grid, dim3(128), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(wkv_prep_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, stack_pdl(), p));
  LinScan s = p.scan;
  const int64_t n = (int64_t)H * dk;
  s.heads = H; s.dk = dk; s.dv = dk; s.share = 1; s.d_scalar = 0; s.read_old = 1;
  s.d = p.f; s.b = p.f + n; s.r = p.f + 2 * n; s.v = p.f + 3 * n; s.bonus = p.f + 4 * n;
  s.p = s.q = s.vscale = nullptr;
  int rc = launch_lin_scan(s, st);
  if (rc != B200_OK) return rc;
  if (dtype == B200_F32) B200_CUDA(launch_pdl(wkv_out_kernel<float>, grid, dim3(128), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(wkv_out_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, stack_pdl(), p));
  return B200_OK;
}

int run_gla(const GlaRun& p, int dtype, cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  const int H = p.a.heads, dk = p.a.dim, dv = p.a.vdim, rk = p.d.rank;
  B200_CHECK_ARG(p.proj && p.f && p.mid && p.scan.n_tok > 0 && p.scan.state && H > 0 && dk > 0 && dv > 0, "gated linear attention: null argument");
  B200_CHECK_ARG(p.d.a2 && p.d.a2_b && p.d.head_norm && p.d.tau > 0.f && rk > 0 && rk <= kGlaMaxRank && dk <= kScanMaxDim,
                 "gated linear attention: null weight, or a bottleneck above %d / a key above %d", kGlaMaxRank, kScanMaxDim);
  const int cw = std::min(kGlaThreads, (dv + 31) / 32 * 32);
  const size_t step_smem = (size_t)(3 * dk + rk + dv + kGlaThreads / cw * cw) * 4;
  if (p.single && step_smem <= 40 * 1024) {
    const dim3 sg(p.scan.n_tok, H);
    if (dtype == B200_F32) B200_CUDA(launch_pdl(gla_step_kernel<float>, sg, dim3(kGlaThreads), step_smem, st, stack_pdl(), p));
    else B200_CUDA(launch_pdl(gla_step_kernel<__nv_bfloat16>, sg, dim3(kGlaThreads), step_smem, st, stack_pdl(), p));
    return B200_OK;
  }
  const int nk = H * dk, nv = H * dv;
  const dim3 pg((p.scan.n_tok + kGlaStrip - 1) / kGlaStrip, (nk + 255) / 256 + (nv + 255) / 256);
  const size_t smem = (size_t)kGlaStrip * rk * 4;
  if (dtype == B200_F32) B200_CUDA(launch_pdl(gla_prep_kernel<float>, pg, dim3(256), smem, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(gla_prep_kernel<__nv_bfloat16>, pg, dim3(256), smem, st, stack_pdl(), p));
  LinScan s = p.scan;
  s.heads = H; s.dk = dk; s.dv = dv; s.share = 1; s.d_scalar = 0; s.d_minus_one = 1;
  s.d = p.f; s.b = p.f + nk; s.r = p.f + 2 * (int64_t)nk; s.v = p.f + 3 * (int64_t)nk;
  s.p = s.q = s.vscale = nullptr;
  int rc = launch_lin_scan(s, st);
  if (rc != B200_OK) return rc;
  const dim3 og((unsigned)(((int64_t)p.scan.n_tok * H + 7) / 8));
  if (dtype == B200_F32) B200_CUDA(launch_pdl(gla_out_kernel<float>, og, dim3(256), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(gla_out_kernel<__nv_bfloat16>, og, dim3(256), 0, st, stack_pdl(), p));
  return B200_OK;
}

int launch_mamba1_conv(const Mamba1Run& p, int dtype, cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  const b200_mamba1_desc& d = p.d;
  B200_CHECK_ARG(p.proj && p.xc && p.slot && p.pos && p.n_tok > 0 && d.inner > 0 && d.conv_w && d.conv_b && d.taps >= 1 && d.taps <= kMambaMaxTaps,
                 "mamba1 convolution: bad arguments (1 … %d taps)", kMambaMaxTaps);
  B200_CHECK_ARG(d.taps == 1 || p.conv_state, "mamba1 convolution: null state");
  if (!p.advance && p.n_tok > kM1Strip && d.taps <= 4 && d.inner % 2 == 0 && p.ld_proj % 2 == 0 && p.off_x % 2 == 0 && p.slot_stride % 2 == 0 &&
      ((reinterpret_cast<uintptr_t>(p.proj) | reinterpret_cast<uintptr_t>(p.xc) | reinterpret_cast<uintptr_t>(p.conv_state) |
        reinterpret_cast<uintptr_t>(d.conv_w) | reinterpret_cast<uintptr_t>(d.conv_b)) & 7) == 0) {
    const dim3 sg((p.n_tok + kM1Strip - 1) / kM1Strip, (d.inner / 2 + 127) / 128);
#define B200_MC(T, TAPS) B200_CUDA(launch_pdl(mamba1_conv_strip_kernel<T, TAPS>, sg, dim3(128), 0, st, stack_pdl(), p))
#define B200_MC_T(T)                    \
  do {                                  \
    if (d.taps == 1) B200_MC(T, 1);     \
    else if (d.taps == 2) B200_MC(T, 2); \
    else if (d.taps == 3) B200_MC(T, 3); \
    else B200_MC(T, 4);                 \
  } while (0)
    if (dtype == B200_F32) B200_MC_T(float);
    else B200_MC_T(__nv_bfloat16);
#undef B200_MC_T
#undef B200_MC
    return B200_OK;
  }
  const dim3 grid(p.n_tok, (d.inner + 127) / 128);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(mamba1_conv_kernel<float>, grid, dim3(128), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(mamba1_conv_kernel<__nv_bfloat16>, grid, dim3(128), 0, st, stack_pdl(), p));
  return B200_OK;
}

int launch_mamba1_dt(const Mamba1Run& p, int dtype, cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  B200_CHECK_ARG(p.xd && p.dt && p.d.w_dt && p.d.dt_b && p.d.dt_rank > 0 && p.n_tok > 0 && p.n_tok <= 65535, "mamba1 step sizes: bad arguments");
  const dim3 grid((p.d.inner + 7) / 8, p.n_tok);
  if (dtype == B200_F32) B200_CUDA(launch_pdl(mamba1_dt_kernel<float>, grid, dim3(256), 0, st, stack_pdl(), p));
  else B200_CUDA(launch_pdl(mamba1_dt_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, stack_pdl(), p));
  return B200_OK;
}

int launch_mamba1_scan(const Mamba1Run& p, int dtype, cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  const b200_mamba1_desc& d = p.d;
  B200_CHECK_ARG(p.xd && p.dt && p.xc && p.proj && p.state && p.mid && p.slot && p.pos && p.n_seg > 0 && p.n_tok > 0 && d.A_log && d.D,
                 "mamba1 scan: null argument");
  B200_CHECK_ARG(d.inner > 0 && d.state > 0 && d.state <= kMamba1MaxState, "mamba1 scan: state 1 … %d", kMamba1MaxState);
#define B200_M1(LPC, NPT)                                                                                                  do {                                                                                                                       const dim3 grid(p.n_seg, (d.inner + 256 / LPC - 1) / (256 / LPC));                                                       if (dtype == B200_F32) B200_CUDA(launch_pdl(mamba1_scan_kernel<float, LPC, NPT>, grid, dim3(256), 0, st, stack_pdl(), p));     else B200_CUDA(launch_pdl(mamba1_scan_kernel<__nv_bfloat16, LPC, NPT>, grid, dim3(256), 0, st, stack_pdl(), p));       } while (0)
  if (d.state <= 8) B200_M1(4, 2);
  else if (d.state <= 16) B200_M1(8, 2);
  else if (d.state <= 32) B200_M1(8, 4);
  else if (d.state <= 64) B200_M1(16, 4);
  else if (d.state <= 128) B200_M1(32, 4);
  else B200_M1(32, 8);
#undef B200_M1
  return B200_OK;
}

int launch_stack_cast_rows(void* y, int64_t ld_y, const float* x, int64_t ld_x, int64_t rows, int n, bool tanh_of, int dtype,
                           cudaStream_t st) {
  REC_DTYPE_CHECK(dtype);
  B200_CHECK_ARG(y && x && rows > 0 && n > 0, "stack cast rows: bad arguments");
  const int64_t total = rows * n;
  const unsigned grid = (unsigned)std::min<int64_t>((total + 255) / 256, 148 * 8);
  if (dtype == B200_F32)
    B200_CUDA(launch_pdl(stack_cast_rows_kernel<float>, dim3(grid), dim3(256), 0, st, stack_pdl(), (float*)y, ld_y, x, ld_x, n, tanh_of ? 1 : 0, total));
  else
    B200_CUDA(launch_pdl(stack_cast_rows_kernel<__nv_bfloat16>, dim3(grid), dim3(256), 0, st, stack_pdl(), (__nv_bfloat16*)y, ld_y, x,
                         ld_x, n, tanh_of ? 1 : 0, total));
  return B200_OK;
}

int launch_stack_rms_add_cast(float* x, const void* y, bool y_bf16, const float* w, __nv_bfloat16* h, int64_t rows, int dim,
                              float eps, float mult, cudaStream_t st) {
  B200_CHECK_ARG(x && y && w && rows > 0 && dim > 0, "stack rms_add_cast: bad arguments");
  if (rows <= 64 && dim <= 16 * 256) {
    if (y_bf16)
      B200_CUDA(launch_pdl(stack_rms_add_cast_small_kernel<__nv_bfloat16>, dim3((unsigned)rows), dim3(256), 0, st, stack_pdl(), x,
                           (const __nv_bfloat16*)y, w, h, dim, eps, mult));
    else
      B200_CUDA(launch_pdl(stack_rms_add_cast_small_kernel<float>, dim3((unsigned)rows), dim3(256), 0, st, stack_pdl(), x,
                           (const float*)y, w, h, dim, eps, mult));
    return B200_OK;
  }
  if (y_bf16)
    B200_CUDA(launch_pdl(stack_rms_add_cast_kernel<__nv_bfloat16>, dim3((unsigned)rows), dim3(256), 0, st, stack_pdl(), x,
                         (const __nv_bfloat16*)y, w, h, dim, eps, mult));
  else
    B200_CUDA(launch_pdl(stack_rms_add_cast_kernel<float>, dim3((unsigned)rows), dim3(256), 0, st, stack_pdl(), x,
                         (const float*)y, w, h, dim, eps, mult));
  return B200_OK;
}

}  // namespace b200

// stack_pool_mma.cu — prompts of the pooled-block attention on the tensor cores (mma.sync m16n8k16 bf16, fp32 accumulate), for
// all sequences of a step that bring enough rows (one grid layer each).  Mixing the heads' softmax weights needs every head's finished weights for the same
// (query, key), so the attention runs in two kernels:
//   pool_stats_kernel   one CTA per (64 query rows, head): the capped scores of all visible keys, online → the row's maximum
//                       and the reciprocal of its denominator (the sink included)
//   pool_mix_kernel     one CTA per (16 query rows, slice of the value columns), all heads: per tile of 16 keys the scores once
//                       more, the finished weights, their mix across heads and the weighted values
// The mix is itself a product, talk [heads × heads] times weights [heads × (query, key) pairs]; the weights enter it as the sum
// of two bf16 numbers (their rounding and what it left), so that it is exact to about 2^-17, and are rounded to bf16 once
// behind it, where they meet the values.  The key list is visited as tiles of block rows, then tiles of token rows.
#include <algorithm>

#include "stack_pool.cuh"

namespace b200 {

namespace {

constexpr float kLog2eM = 1.4426950408889634f;

__device__ __forceinline__ void cp16(void* dst, const void* src, bool live) {   // dead chunks are filled with zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ float ex2(float x) {   // relative error about 2^-22; 2^(−inf) = 0
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// A raw dot product → the capped score times log2(e).  cap·tanh(z) as cap·(1 − 2 / (1 + e^(2z))): an absolute error of about
// 1e-7·cap, which is what the softmax sees.
struct ScoreMap {
  float in, out;   // capped: 2^(s·in) = e^(2·s·scale/cap), out = cap·log2 e;  uncapped: in = 0, out = scale·log2 e
};
__device__ __forceinline__ float map_score(float s, const ScoreMap& m) {
  if (m.in == 0.f) return s * m.out;
  const float e = ex2(fminf(s * m.in, 126.f));
  return fmaf(-2.f * m.out, rcp(1.f + e), m.out);
}

struct PoolMma {
  PoolAttn p{};                  // the step's rows
  const int32_t *seg_row0 = nullptr, *seg_count = nullptr;
  int min_rows = 1;              // sequences with fewer rows are left to other kernels
  ScoreMap map{};
  float* stats = nullptr;        // [n_tok][heads][2]: maximum (log2 units), 1 / denominator
  int vcols = 0, kstages = 1;    // pool_mix_kernel: value columns per CTA, key tiles in shared memory
};
// one sequence's rows and cache
struct SeqView {
  int row0, count, pos0;
  const __nv_bfloat16 *k, *v;
};
__device__ __forceinline__ SeqView seq_view(const PoolMma& m, int seg) {
  SeqView s;
  s.row0 = m.seg_row0[seg];
  s.count = m.seg_count[seg];
  s.pos0 = m.p.pos[s.row0];
  const int64_t slot = m.p.slot[s.row0];
  s.k = static_cast<const __nv_bfloat16*>(m.p.kcache) + slot * m.p.k_slot_stride;
  s.v = static_cast<const __nv_bfloat16*>(m.p.vcache) + slot * m.p.v_slot_stride;
  return s;
}

// The keys a tile of rows at positions [p0, p1] may see: blocks [0, nb) and tokens [lo, p1].
struct TileList {
  int nb, lo, p1, block_tiles, tiles;
};
template <int BN>
__device__ __forceinline__ TileList tile_list(const PoolAttn& p, int p0, int p1) {
  TileList t;
  t.nb = pool_nb(p1, p.a.window, p.d.pool);
  t.lo = pool_lo(p0, p.a.window);
  t.p1 = p1;
  t.block_tiles = (t.nb + BN - 1) / BN;
  t.tiles = t.block_tiles + (p1 - t.lo + BN) / BN;
  return t;
}
// first cache row of tile `it`, and how many of its rows are in the list
__device__ __forceinline__ int tile_row0(const TileList& t, int it, int bn, int max_ctx, int& n) {
  if (it < t.block_tiles) {
    n = t.nb - it * bn;
    return max_ctx + it * bn;
  }
  const int j0 = t.lo + (it - t.block_tiles) * bn;
  n = t.p1 - j0 + 1;
  return j0;
}

// ------------------------------------------------------------------------------------------------------------ statistics
constexpr int kStM = 64, kStN = 64;
template <int KS>   // dim / 16
__global__ void __launch_bounds__(128) pool_stats_kernel(const PoolMma m) {
  extern __shared__ __align__(128) uint8_t ps_smem[];
  constexpr int LD = KS * 32 + 16;   // bytes per staged row: an odd number of 16-byte chunks, conflict-free for ldmatrix
  const PoolAttn& p = m.p;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int h = blockIdx.y, H = p.a.heads, G = p.a.kv_heads, dk = KS * 16, kvh = h / (H / G);
  const SeqView sv = seq_view(m, blockIdx.z);
  const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kStM;   // rows with the most keys first
  if (q0 >= sv.count || sv.count < m.min_rows) return;
  const int rows = min(kStM, sv.count - q0);
  uint8_t* Qs = ps_smem;                  // [64][LD]
  uint8_t* Ks = Qs + kStM * LD;           // [2][64][LD]
  const TileList tl = tile_list<kStN>(p, sv.pos0 + q0, sv.pos0 + q0 + rows - 1);
  const __nv_bfloat16* qg = static_cast<const __nv_bfloat16*>(p.q) + (int64_t)sv.row0 * H * dk + (int64_t)h * dk;
  const __nv_bfloat16* kg = sv.k + (int64_t)kvh * dk;
  constexpr int CH = KS * 2;
  for (int i = tid; i < kStM * CH; i += 128) {
    const int r = i / CH, c = i % CH;
    cp16(Qs + r * LD + c * 16, qg + (int64_t)min(q0 + r, sv.count - 1) * H * dk + c * 8, r < rows);
  }
  auto load = [&](int it) {
    int n;
    const int r0 = tile_row0(tl, it, kStN, p.max_ctx, n);
    uint8_t* dst = Ks + (it & 1) * kStN * LD;
    for (int i = tid; i < kStN * CH; i += 128) {
      const int r = i / CH, c = i % CH;
      cp16(dst + r * LD + c * 16, kg + (int64_t)(r0 + min(r, n - 1)) * G * dk + c * 8, r < n);
    }
    cp_commit();
  };
  load(0);
  uint32_t qf[KS][4];
  const int i0 = sv.pos0 + q0 + warp * 16 + g, i1 = i0 + 8;
  const int lo0 = pool_lo(i0, p.a.window), lo1 = pool_lo(i1, p.a.window);
  const int nb0 = pool_nb(i0, p.a.window, p.d.pool), nb1 = pool_nb(i1, p.a.window, p.d.pool);
  float mx0 = -INFINITY, mx1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  for (int it = 0; it < tl.tiles; ++it) {
    cp_wait<0>();
    __syncthreads();   // tile `it` is there, and everyone is done with the buffer the next load writes
    if (it + 1 < tl.tiles) load(it + 1);
    if (it == 0) {
#pragma unroll
      for (int k = 0; k < KS; ++k)
        ldsm4(smem_u32(Qs + (warp * 16 + (lane & 15)) * LD + k * 32 + (lane >> 4) * 16), qf[k]);
    }
    const uint8_t* K = Ks + (it & 1) * kStN * LD;
    const bool blk = it < tl.block_tiles;
    const int j0 = blk ? it * kStN : tl.lo + (it - tl.block_tiles) * kStN;
    // visible keys of the two rows as ranges of in-tile columns
    const int a0 = blk ? 0 : lo0 - j0, e0 = blk ? nb0 - j0 : i0 - j0 + 1;
    const int a1 = blk ? 0 : lo1 - j0, e1 = blk ? nb1 - j0 : i1 - j0 + 1;
    float s[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; nt += 2) {
#pragma unroll
      for (int x = 0; x < 4; ++x) s[nt][x] = s[nt + 1][x] = 0.f;
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        uint32_t b[4];   // keys nt·8 … + 7: entries 0-7 and 8-15; keys + 8 … + 15: the same
        ldsm4(smem_u32(K + (nt * 8 + (lane & 7) + (lane >> 4) * 8) * LD + k * 32 + ((lane >> 3) & 1) * 16), b);
        mma16816(s[nt], qf[k], b[0], b[1]);
        mma16816(s[nt + 1], qf[k], b[2], b[3]);
      }
    }
    float t0 = -INFINITY, t1 = -INFINITY;
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int c = nt * 8 + tq * 2 + x;
        s[nt][x] = c >= a0 && c < e0 ? map_score(s[nt][x], m.map) : -INFINITY;
        s[nt][x + 2] = c >= a1 && c < e1 ? map_score(s[nt][x + 2], m.map) : -INFINITY;
        t0 = fmaxf(t0, s[nt][x]);
        t1 = fmaxf(t1, s[nt][x + 2]);
      }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) {
      t0 = fmaxf(t0, __shfl_xor_sync(0xffffffffu, t0, o));
      t1 = fmaxf(t1, __shfl_xor_sync(0xffffffffu, t1, o));
    }
    const float n0 = fmaxf(mx0, t0), n1 = fmaxf(mx1, t1);
    const float b0 = n0 == -INFINITY ? 0.f : n0, b1 = n1 == -INFINITY ? 0.f : n1;   // nothing seen yet: 2^(−inf − 0) = 0
    l0 *= ex2(mx0 - b0);
    l1 *= ex2(mx1 - b1);
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        l0 += ex2(s[nt][x] - b0);
        l1 += ex2(s[nt][x + 2] - b1);
      }
    mx0 = n0;
    mx1 = n1;
  }
#pragma unroll
  for (int o = 1; o < 4; o <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, o);
    l1 += __shfl_xor_sync(0xffffffffu, l1, o);
  }
  if (tq != 0) return;
  const float sink = p.d.sink != nullptr ? p.d.sink[h] * kLog2eM : -INFINITY;
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int r = q0 + warp * 16 + g + 8 * x;
    if (r >= sv.count) continue;
    const float mx = x ? mx1 : mx0, l = x ? l1 : l0, mm = fmaxf(mx, sink);   // a row always sees itself: mx is finite
    float* o = m.stats + ((int64_t)(sv.row0 + r) * H + h) * 2;
    o[0] = mm;
    o[1] = 1.f / (l * ex2(mx - mm) + ex2(sink - mm));
  }
}

// ------------------------------------------------------------------------------------------------- mixed weights, values
// Warp w owns heads w·HPW … w·HPW + HPW − 1 for the scores and the values, and every NW-th group of eight (key, query) pairs
// for the mix.  HPW 1: up to 16 heads; 2: up to 32, and half as many value columns per CTA.  Shared layouts (16-bit entries;
// strides padded so that ldmatrix and the scattered stores meet few bank conflicts):
//   weights  [key 16][query 16][head] words {low part, high part} — the mix reads eight pairs × eight heads as its B operand of
//            sixteen columns, against a mixing matrix that has every column twice
//   mixed    [head][key 16][query 16] — the values read it transposed as their A operand
// The tiles run through two phases: the scores and weights of tile t + 1 beside the values of tile t, then the mix of tile
// t + 1.  Keys and values of later tiles are on their way meanwhile.
template <int HPW> struct MixShape {
  static constexpr int KH = HPW;                          // head groups of 16
  static constexpr int PW = 16 * KH + 4;                  // words per pair
  static constexpr int JW = 16 * PW + 1;                  // words per key
  static constexpr int WBYTES = (16 * JW * 4 + 15) / 16 * 16;
  static constexpr int XW = 196;                          // words per head of the mixed weights: 16 rows of 12 words, + 4
  static constexpr int XBYTES = 16 * KH * XW * 4;
  static constexpr int NT = 16 / HPW;                     // most 8-column tiles of a CTA's slice of the values
};
__host__ __device__ inline int mix_smem(int H, int G, int dk, int vcols, int kstages, int wbytes, int xbytes) {
  return 16 * (H * dk * 2 + 16) + 16 * (kstages * (G * dk * 2 + 16) + 2 * (G * vcols * 2 + 16)) + wbytes + xbytes;
}

// KS: dim / 16 and the CTA's whole NT column tiles, known at compile time; 0: any size.
template <int HPW, int KS>
__global__ void __launch_bounds__(512, 1) pool_mix_kernel(const PoolMma m) {
  extern __shared__ __align__(128) uint8_t pm_smem[];
  using SH = MixShape<HPW>;
  constexpr int KH = SH::KH;
  const PoolAttn& p = m.p;
  const int tid = threadIdx.x, nthr = blockDim.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3, nw = nthr >> 5;
  const int H = p.a.heads, G = p.a.kv_heads, per = H / G, dk = p.a.dim, dv = p.a.vdim, ks = KS > 0 ? KS : dk / 16;
  const SeqView sv = seq_view(m, blockIdx.z);
  const int q0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * 16, rows = min(16, sv.count - q0);
  if (rows <= 0 || sv.count < m.min_rows) return;
  const int c0 = blockIdx.y * m.vcols, vc = min(m.vcols, dv - c0), nt_v = KS > 0 ? SH::NT : vc / 8;
  const int ldq = H * dk * 2 + 16, ldk = G * dk * 2 + 16, ldv = G * m.vcols * 2 + 16;
  uint8_t* Qs = pm_smem;
  uint8_t* Ks = Qs + 16 * ldq;
  uint8_t* Vs = Ks + m.kstages * 16 * ldk;
  uint32_t* W = reinterpret_cast<uint32_t*>(Vs + 2 * 16 * ldv);
  uint32_t* X = W + SH::WBYTES / 4;
  const TileList tl = tile_list<16>(p, sv.pos0 + q0, sv.pos0 + q0 + rows - 1);
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q) + (int64_t)sv.row0 * H * dk;
    const int ch = H * dk / 8;
    for (int i = tid; i < 16 * ch; i += nthr) {
      const int r = i / ch, c = i % ch;
      cp16(Qs + r * ldq + c * 16, q + (int64_t)min(q0 + r, sv.count - 1) * H * dk + c * 8, r < rows);
    }
  }
  // a warp copies whole rows, so that no index is divided per chunk; the columns of a slice of the values lie vch1 chunks per
  // key/value head apart (the reciprocal is exact for the few hundred chunks of a row)
  const int kch = G * dk / 8, vch1 = vc / 8, vch = G * vch1, vmagic = (65536 + vch1 - 1) / vch1;
  auto k_buf = [&](int it) { return Ks + (m.kstages == 2 ? it & 1 : 0) * 16 * ldk; };
  auto v_buf = [&](int it) { return Vs + (it & 1) * 16 * ldv; };
  const int64_t krow = (int64_t)G * dk, vrow = (int64_t)G * dv;
  const __nv_bfloat16* k_src = sv.k + lane * 8;
  const __nv_bfloat16* v_src = sv.v + c0;
  const bool v_whole = vc == dv;   // the slice is the whole row: one run of chunks
  auto load_k = [&](int it) {
    if (it >= tl.tiles) return;
    int n;
    const int r0 = tile_row0(tl, it, 16, p.max_ctx, n);
    uint8_t* d = k_buf(it) + lane * 16;
    for (int r = warp; r < 16; r += nw) {
      const __nv_bfloat16* kr = k_src + (int64_t)(r0 + min(r, n - 1)) * krow;
#pragma unroll 4
      for (int c = 0; c + lane < kch; c += 32) cp16(d + r * ldk + c * 16, kr + c * 8, r < n);
    }
  };
  auto load_v = [&](int it) {
    if (it >= tl.tiles) return;
    int n;
    const int r0 = tile_row0(tl, it, 16, p.max_ctx, n);
    uint8_t* d = v_buf(it);
    for (int r = warp; r < 16; r += nw) {
      const __nv_bfloat16* vr = v_src + (int64_t)(r0 + min(r, n - 1)) * vrow;
      if (v_whole) {
#pragma unroll 4
        for (int e = lane; e < vch; e += 32) cp16(d + r * ldv + e * 16, vr + e * 8, r < n);
        continue;
      }
      for (int e = lane; e < vch; e += 32) {
        const int gg = (e * vmagic) >> 16, c = e - gg * vch1;
        cp16(d + r * ldv + gg * m.vcols * 2 + c * 16, vr + gg * dv + c * 8, r < n);
      }
    }
  };
  load_k(0);
  load_v(0);
  if (m.kstages == 2) load_k(1);
  cp_commit();
  // heads that do not exist keep zero weights
  for (int i = tid; i < SH::WBYTES / 4; i += nthr) W[i] = 0;
  // the mixing matrix as A fragments: rows = mixed head, columns 2h and 2h + 1 = head h
  uint32_t tf[KH][2 * KH][4];
  {
    auto talk = [&](int a, int b) {
      if (a >= H || b >= H) return 0.f;
      return p.d.talk != nullptr ? p.d.talk[a * H + b] : a == b ? 1.f : 0.f;
    };
#pragma unroll
    for (int a = 0; a < KH; ++a)
#pragma unroll
      for (int b = 0; b < 2 * KH; ++b)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const float v = talk(a * 16 + g + (x & 1) * 8, b * 8 + tq + (x >> 1) * 4);
          tf[a][b][x] = pack2(v, v);
        }
  }
  const int i0 = sv.pos0 + q0 + g, i1 = i0 + 8, nb0 = pool_nb(i0, p.a.window, p.d.pool), nb1 = pool_nb(i1, p.a.window, p.d.pool);
  const int nb_first = pool_nb(sv.pos0 + q0, p.a.window, p.d.pool), lo_last = pool_lo(sv.pos0 + q0 + 15, p.a.window);
  float mx[HPW][2], il[HPW][2], o[HPW][SH::NT][4];
#pragma unroll
  for (int u = 0; u < HPW; ++u) {
    const int h = warp * HPW + u;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int r = q0 + g + 8 * x;
      const bool live = h < H && r < sv.count;
      mx[u][x] = live ? m.stats[((int64_t)(sv.row0 + r) * H + h) * 2] : 0.f;
      il[u][x] = live ? m.stats[((int64_t)(sv.row0 + r) * H + h) * 2 + 1] : 0.f;
    }
#pragma unroll
    for (int n = 0; n < SH::NT; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) o[u][n][x] = 0.f;
  }
  float s[HPW][2][4];
  // raw scores of tile `it`, this warp's heads
  auto scores = [&](int it) {
    const uint8_t* K = k_buf(it);
#pragma unroll
    for (int u = 0; u < HPW; ++u) {
      const int h = warp * HPW + u;
#pragma unroll
      for (int x = 0; x < 4; ++x) s[u][0][x] = s[u][1][x] = 0.f;
      if (h >= H) break;
      const uint32_t qa = smem_u32(Qs + (lane & 15) * ldq + h * dk * 2 + (lane >> 4) * 16);
      const uint32_t ka = smem_u32(K + ((lane & 7) + (lane >> 4) * 8) * ldk + (h / per) * dk * 2 + ((lane >> 3) & 1) * 16);
#pragma unroll(KS > 0 ? KS : 2)
      for (int k = 0; k < ks; ++k) {
        uint32_t a[4], b[4];   // b: keys 0-7, entries 0-7 and 8-15; keys 8-15, the same
        ldsm4(qa + k * 32, a);
        ldsm4(ka + k * 32, b);
        mma16816(s[u][0], a, b[0], b[1]);
        mma16816(s[u][1], a, b[2], b[3]);
      }
    }
  };
  // … → finished weights in W
  uint32_t* Wt = W + tq * 2 * SH::JW + g * SH::PW;
  auto weights = [&](int it) {
    const bool blk = it < tl.block_tiles;
    const int j0 = blk ? it * 16 : tl.lo + (it - tl.block_tiles) * 16;
    // tiles every row sees whole need no mask: keys from the last row's window edge to the first row's position, or blocks the
    // first row sees
    const bool whole = blk ? j0 + 16 <= nb_first : j0 >= lo_last && j0 + 15 <= sv.pos0 + q0;
    int a0 = 0, e0 = 16, a1 = 0, e1 = 16;   // visible keys of the two rows as ranges of in-tile columns
    if (!whole) {
      a0 = blk ? 0 : pool_lo(i0, p.a.window) - j0;
      a1 = blk ? 0 : pool_lo(i1, p.a.window) - j0;
      e0 = (blk ? nb0 : i0 + 1) - j0;
      e1 = (blk ? nb1 : i1 + 1) - j0;
    }
#pragma unroll
    for (int u = 0; u < HPW; ++u) {
      const int h = warp * HPW + u;
      if (h >= H) break;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          float w = ex2(map_score(s[u][nt][x], m.map) - mx[u][x >> 1]) * il[u][x >> 1];
          if (!whole) {
            const int j = nt * 8 + tq * 2 + (x & 1);
            if (!((x >> 1) ? j >= a1 && j < e1 : j >= a0 && j < e0)) w = 0.f;
          }
          const float hi = __uint_as_float(__float_as_uint(w) & 0xffff0000u);   // the upper half is a bf16 number as it is
          Wt[(nt * 8 + (x & 1)) * SH::JW + (x >> 1) * 8 * SH::PW + h] = pack2(w - hi, hi);
        }
    }
  };
  // W → mixed weights in X, eight pairs (one key, queries iq …) at a time
  auto mixed = [&]() {
    const int iq = (warp & 1) * 8;   // the number of warps is even
    const uint32_t* w = W + (warp >> 1) * SH::JW + (iq + g) * SH::PW + tq;
    uint32_t* d = X + g * SH::XW + (warp >> 1) * 12 + (iq >> 1) + tq;
    for (int nt = warp; nt < 32; nt += nw, w += (nw >> 1) * SH::JW, d += (nw >> 1) * 12) {
      float x[KH][4];
#pragma unroll
      for (int a = 0; a < KH; ++a)
#pragma unroll
        for (int e = 0; e < 4; ++e) x[a][e] = 0.f;
#pragma unroll
      for (int b = 0; b < 2 * KH; ++b) {
        const uint32_t w0 = w[b * 8], w1 = w[b * 8 + 4];
#pragma unroll
        for (int a = 0; a < KH; ++a) mma16816(x[a], tf[a][b], w0, w1);
      }
#pragma unroll
      for (int a = 0; a < KH; ++a) {
        d[a * 16 * SH::XW] = pack2(x[a][0], x[a][1]);
        d[(a * 16 + 8) * SH::XW] = pack2(x[a][2], x[a][3]);
      }
    }
  };
  // mixed weights of tile `it` times its values
  auto values = [&](int it) {
    const uint8_t* V = v_buf(it);
#pragma unroll
    for (int u = 0; u < HPW; ++u) {
      const int h = warp * HPW + u;
      if (h >= H) break;
      uint32_t a[4];   // stored [key][query]: matrices (keys 0-7, queries 0-7), (keys 0-7, queries 8-15), (keys 8-15, …), …
      ldsm4_t(smem_u32(X + h * SH::XW + ((lane & 7) + (lane >> 4) * 8) * 12) + ((lane >> 3) & 1) * 16, a);
      const uint32_t va = smem_u32(V + (lane & 15) * ldv + (h / per) * m.vcols * 2 + (lane >> 4) * 16);
#pragma unroll
      for (int n = 0; n < SH::NT; n += 2) {
        if (KS == 0 && n >= nt_v) break;
        uint32_t b[4];   // columns n·8 … + 7: keys 0-7 and 8-15; columns + 8 … + 15: the same
        ldsm4_t(va + n * 16, b);
        mma16816(o[u][n], a, b[0], b[1]);
        mma16816(o[u][n + 1], a, b[2], b[3]);
      }
    }
  };
  cp_wait<0>();
  __syncthreads();
  scores(0);
  weights(0);
  __syncthreads();
  if (m.kstages == 1) {
    load_k(1);
    cp_commit();
  }
  mixed();
  cp_wait<0>();
  __syncthreads();
  for (int it = 0; it < tl.tiles; ++it) {
    const bool more = it + 1 < tl.tiles;
    load_v(it + 1);
    if (m.kstages == 2) load_k(it + 2);
    cp_commit();
    if (more) scores(it + 1);
    values(it);
    if (!more) break;
    weights(it + 1);
    __syncthreads();   // every weight of tile it + 1 is in W; tile it's values and mixed weights have been read
    if (m.kstages == 1) {
      load_k(it + 2);
      cp_commit();
    }
    mixed();
    cp_wait<0>();
    __syncthreads();   // mixed weights, and the next keys and values
  }
#pragma unroll
  for (int u = 0; u < HPW; ++u) {
    const int h = warp * HPW + u;
    if (h >= H) break;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int r = q0 + g + 8 * x;
      if (r >= sv.count) continue;
      __nv_bfloat16* y = static_cast<__nv_bfloat16*>(p.mid) + (int64_t)(sv.row0 + r) * p.ld_mid + h * dv + c0 + tq * 2;
#pragma unroll
      for (int n = 0; n < SH::NT; ++n)
        if (n < nt_v)
          *reinterpret_cast<uint32_t*>(y + n * 8) = pack2(o[u][n][2 * x] * p.out_scale, o[u][n][2 * x + 1] * p.out_scale);
    }
  }
}

template <int KS>
int launch_stats(const PoolMma& m, int n_seg, int max_count, cudaStream_t st) {
  constexpr int smem = 3 * 64 * (KS * 32 + 16);
  if (smem > 48 * 1024) {
    static bool attr_done = false;
    if (!attr_done) {
      B200_CUDA(cudaFuncSetAttribute(pool_stats_kernel<KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
      attr_done = true;
    }
  }
  const dim3 grid((max_count + kStM - 1) / kStM, m.p.a.heads, n_seg);
  B200_CUDA(launch_pdl(pool_stats_kernel<KS>, grid, dim3(128), (size_t)smem, st, false, m));
  return B200_OK;
}

template <int HPW, int KS>
int launch_mix(PoolMma m, int n_seg, int max_count, cudaStream_t st) {
  using SH = MixShape<HPW>;
  const b200_attn_desc& a = m.p.a;
  static bool attr_done = false;
  if (!attr_done) {
    B200_CUDA(cudaFuncSetAttribute(pool_mix_kernel<HPW, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    attr_done = true;
  }
  const int splits = (a.vdim + SH::NT * 8 - 1) / (SH::NT * 8);
  m.vcols = ((a.vdim + splits - 1) / splits + 15) / 16 * 16;
  m.kstages = mix_smem(a.heads, a.kv_heads, a.dim, m.vcols, 2, SH::WBYTES, SH::XBYTES) <= 227 * 1024 ? 2 : 1;
  const int smem = mix_smem(a.heads, a.kv_heads, a.dim, m.vcols, m.kstages, SH::WBYTES, SH::XBYTES);
  const int warps = std::max(4, ((a.heads + HPW - 1) / HPW + 1) / 2 * 2);
  const dim3 grid((max_count + 15) / 16, (a.vdim + m.vcols - 1) / m.vcols, n_seg);
  B200_CUDA(launch_pdl(pool_mix_kernel<HPW, KS>, grid, dim3(warps * 32), (size_t)smem, st, false, m));
  return B200_OK;
}

}  // namespace

bool pool_prompt_ok(const b200_attn_desc& a) {
  if (a.heads > 32 || a.dim % 16 != 0 || a.dim > 128 || a.vdim % 16 != 0 || a.vdim > 256) return false;
  const int vmax = a.heads <= 16 ? 128 : 64, splits = (a.vdim + vmax - 1) / vmax, vc = ((a.vdim + splits - 1) / splits + 15) / 16 * 16;
  const int w = a.heads <= 16 ? MixShape<1>::WBYTES : MixShape<2>::WBYTES, x = a.heads <= 16 ? MixShape<1>::XBYTES : MixShape<2>::XBYTES;
  return mix_smem(a.heads, a.kv_heads, a.dim, vc, 1, w, x) <= 227 * 1024;
}

int launch_pool_prompt(const PoolAttn& p, const int32_t* seg_row0, const int32_t* seg_count, int n_seg, int max_count, int min_rows, float* stats,
                       cudaStream_t st) {
  const b200_attn_desc& a = p.a;
  B200_CHECK_ARG(p.q && p.kcache && p.vcache && p.mid && stats && seg_row0 && seg_count && p.slot && p.pos && n_seg > 0 && max_count > 0,
                 "pool prompt attention: bad arguments");
  B200_CHECK_ARG(pool_prompt_ok(a) && a.heads % a.kv_heads == 0, "pool prompt attention: head sizes not built");
  B200_CHECK_ARG(((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.kcache) | reinterpret_cast<uintptr_t>(p.vcache)) & 15) == 0 &&
                     p.k_slot_stride % 8 == 0 && p.v_slot_stride % 8 == 0 && p.ld_mid % 2 == 0 && (reinterpret_cast<uintptr_t>(p.mid) & 3) == 0,
                 "pool prompt attention: operands must be 16-byte aligned");
  PoolMma m;
  m.p = p; m.seg_row0 = seg_row0; m.seg_count = seg_count; m.min_rows = min_rows; m.stats = stats;
  if (p.d.softcap > 0.f) {
    m.map.in = 2.f * a.scale / p.d.softcap * kLog2eM;
    m.map.out = p.d.softcap * kLog2eM;
  } else {
    m.map.out = a.scale * kLog2eM;
  }
  int rc = B200_OK;
  switch (a.dim / 16) {
    case 1: rc = launch_stats<1>(m, n_seg, max_count, st); break;
    case 2: rc = launch_stats<2>(m, n_seg, max_count, st); break;
    case 3: rc = launch_stats<3>(m, n_seg, max_count, st); break;
    case 4: rc = launch_stats<4>(m, n_seg, max_count, st); break;
    case 5: rc = launch_stats<5>(m, n_seg, max_count, st); break;
    case 6: rc = launch_stats<6>(m, n_seg, max_count, st); break;
    case 7: rc = launch_stats<7>(m, n_seg, max_count, st); break;
    default: rc = launch_stats<8>(m, n_seg, max_count, st); break;
  }
  if (rc != B200_OK) return rc;
  const bool k8 = a.dim == 128 && a.vdim == 128;
  if (a.heads <= 16) return k8 ? launch_mix<1, 8>(m, n_seg, max_count, st) : launch_mix<1, 0>(m, n_seg, max_count, st);
  return k8 ? launch_mix<2, 8>(m, n_seg, max_count, st) : launch_mix<2, 0>(m, n_seg, max_count, st);
}

}  // namespace b200

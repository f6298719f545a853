// Attention of all query heads of a request over its cached latent rows: every head's query has already been multiplied by
// the head's key up-projection, so one row [c | turned key part] per token serves all heads as key (the whole row) and as
// value (its c part), and a row is read once per 16 (token, head) pairs instead of once per head.
// A CTA of sixteen warps owns 16 query rows - consecutive (token, head) pairs of one request - and walks its part of the
// visible keys in tiles of 64, which a seventeenth warp brings into shared memory in halves of 32 by TMA (swizzled boxes of 64 columns):
//   S = Q K^T   mma.sync m16n8k16, each warp every eighth 16-column step of half the keys (its part of Q stays in registers),
//               the warps' fp32 parts summed through shared memory
//   softmax     one row per warp, two keys per lane: window mask, running maximum and sum in fp32, P in bfloat16
//   O += P C    each warp its share of the kv_rank columns, fp32 accumulators in registers
// Decode steps split the key range over several CTAs (too few requests to fill the GPU otherwise); the CTA
// that finishes last merges their (m, l, O) and adds the sink's share of the denominator.  HBM-bound: a row's bytes are used for 2 * 16 heads' flops.
#include <cuda.h>

#include <algorithm>

#include "common.cuh"
#include "hybrid_ops.h"

namespace kge {
inline namespace b16 {
int make_tmap(CUtensorMap* m, const void* ptr, int64_t rows, int64_t cols, int box_rows);      // gemm_tc.cu: boxes of 64 columns, 128-byte swizzle
}

namespace {

constexpr int LM_WARPS = 16, LM_KW = 8, LM_KH = 32, LM_KT = 2 * LM_KH, LM_ROWS = 16, LM_KSW = 5;      // LM_KW: warps that share a row's columns; LM_KSW: 16-column steps per warp at most
constexpr float LM_LOG2E = 1.4426950408889634f;
typedef __nv_bfloat16 lm_bf16;

__device__ __forceinline__ uint32_t lm_saddr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void lm_mbar_init(uint32_t bar, uint32_t count) { asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count)); }
__device__ __forceinline__ void lm_mbar_arrive(uint32_t bar) { asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory"); }
__device__ __forceinline__ void lm_mbar_expect(uint32_t bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
// false when the phase has not completed within a second or so (the caller goes on and marks its results)
__device__ __forceinline__ bool lm_mbar_wait(uint32_t bar, uint32_t parity) {
  uint32_t ok = 0;
  for (uint32_t spin = 0; spin < (1u << 24); ++spin) {
    asm volatile("{\n.reg .pred p;\nmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\nselp.u32 %0, 1, 0, p;\n}" : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
    if (ok) return true;
  }
  return false;
}
__device__ __forceinline__ void lm_tma(uint32_t dst, const CUtensorMap* map, uint32_t bar, int c0, int c1) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];" ::"r"(dst), "l"(map), "r"(bar), "r"(c0), "r"(c1) : "memory");
}
__device__ __forceinline__ void lm_sync() { asm volatile("bar.sync 1, 512;" ::: "memory"); }      // the sixteen computing warps
__device__ __forceinline__ void lm_ldm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void lm_ldm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void lm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ float lm_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

constexpr int LM_BLK = LM_KH * 128;                    // a stage is blocks of 32 rows x 64 columns, 16-byte pieces XOR-swizzled by row % 8
constexpr int LM_SLD = LM_KT + 4, LM_PLD = LM_KT + 8;
size_t lm_smem(int dim, int st) {
  return 1024 + (size_t)st * ((dim + 63) / 64) * LM_BLK + (size_t)LM_KW * LM_ROWS * LM_SLD * 4 + (size_t)LM_ROWS * LM_PLD * 2 + 3 * LM_ROWS * 4 + (size_t)2 * st * 8;
}

constexpr int LM_COUNTERS = 256;                            // arrival counters of the row tiles, ahead of the parts in the workspace (at most 74: two parts or more of each share 148 SMs)

// VP: 16-column pairs of the output per warp; ST: stages of 32 keys (two are computed on, the others in flight)
template <int VP, int ST>
__global__ void __launch_bounds__(LM_WARPS * 32 + 32) latent_mqa_kernel(const __grid_constant__ CUtensorMap tm, LatentMqaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) unsigned char lm_raw[];
  const int dim = a.kv_rank + a.rot_part, H = a.H, blocks = (dim + 63) >> 6;
  const uint32_t stage_bytes = (uint32_t)(blocks * LM_BLK), sK = (lm_saddr(lm_raw) + 1023u) & ~1023u;      // swizzled boxes start on 1024 bytes
  float* Ss = reinterpret_cast<float*>(lm_raw + (sK - lm_saddr(lm_raw)) + ST * stage_bytes);     // [8][16][64]: the warps' parts of the scores
  lm_bf16* Ps = reinterpret_cast<lm_bf16*>(Ss + LM_KW * LM_ROWS * LM_SLD);
  float* cs = reinterpret_cast<float*>(Ps + LM_ROWS * LM_PLD);      // [16] correction of this tile, then [16] m, [16] l
  const uint32_t bars = lm_saddr(cs + 3 * LM_ROWS);                  // [ST] full, [ST] empty
  auto full = [&](int i) { return bars + 8u * i; };
  auto empty = [&](int i) { return bars + 8u * (ST + i); };
  const int b = a.req0 + blockIdx.z, rs = a.qsl[b], nrows = (a.qsl[b + 1] - rs) * H, R0 = blockIdx.x * LM_ROWS;
  if (R0 >= nrows) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos_first = a.positions[rs + R0 / H], pos_last = a.positions[rs + min(R0 + LM_ROWS - 1, nrows - 1) / H];
  const int lo_min = a.window > 0 ? max(0, pos_first - a.window + 1) / LM_KT * LM_KT : 0;      // whole tiles: a stage lies inside a page
  const int ntiles = (pos_last - lo_min) / LM_KT + 1, per = (ntiles + a.splits - 1) / a.splits;
  const int t0 = blockIdx.y * per, t1 = min(ntiles, t0 + per);
  const int bs_shift = 31 - __clz(a.block_size);
  const int32_t* bt = a.block_table + (int64_t)b * a.max_blocks;
  if (tid == 0) {
    for (int i = 0; i < ST; ++i) { lm_mbar_init(full(i), 1); lm_mbar_init(empty(i), LM_WARPS); }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  if (warp == LM_WARPS) {
    // the copying thread: a stage is one box per 64 columns (and per page, where pages are shorter than a stage).  Rows beyond
    // the last key are other rows of its page: finite numbers that the mask keeps out.
    if (lane == 0) {
      const int brows = min(a.block_size, LM_KH), nb = LM_KH / brows, last_page = pos_last >> bs_shift;
      int slot = 0;
      uint32_t phase = 1;                             // the first pass finds every stage empty
      int pg = bt[min((lo_min + 2 * t0 * LM_KH) >> bs_shift, last_page)];
      for (int hk = 2 * t0; hk < 2 * t1; ++hk) {
        const int next = bt[min((lo_min + (hk + 1) * LM_KH) >> bs_shift, last_page)];      // requested a stage ahead
        if (!lm_mbar_wait(empty(slot), phase)) return;
        lm_mbar_expect(full(slot), stage_bytes);
        for (int r = 0; r < nb; ++r) {
          const int j = lo_min + hk * LM_KH + r * brows;
          const int page = r == 0 ? pg : bt[min(j >> bs_shift, last_page)];
          const int row = (page << bs_shift) + (j & (a.block_size - 1));
          for (int c = 0; c < blocks; ++c) lm_tma(sK + slot * stage_bytes + c * LM_BLK + r * brows * 128, &tm, full(slot), c * 64, row);
        }
        pg = next;
        if (++slot == ST) { slot = 0; phase ^= 1; }
      }
    }
    return;
  }
  // a warp takes 32 of a tile's 64 keys and every eighth 16-column step of their rows
  const int kw = warp % LM_KW, half = warp / LM_KW;
  // its steps (kw, kw + 8, ..) of the 16 query rows, as A fragments (rows beyond the request's repeat its last one; they are never written)
  const int ksteps = dim >> 4, vpairs = a.kv_rank >> 4;
  uint32_t qf[LM_KSW][4];
  {
    const lm_bf16* q = (const lm_bf16*)a.q + (int64_t)rs * H * dim + (lane & 3) * 2;
    const lm_bf16 *q0 = q + (int64_t)min(R0 + (lane >> 2), nrows - 1) * dim, *q1 = q + (int64_t)min(R0 + (lane >> 2) + 8, nrows - 1) * dim;
#pragma unroll
    for (int i = 0; i < LM_KSW; ++i) {
      const int c = (kw + i * LM_KW) * 16;
      const bool in = c < dim;
      qf[i][0] = in ? *reinterpret_cast<const uint32_t*>(q0 + c) : 0u;
      qf[i][1] = in ? *reinterpret_cast<const uint32_t*>(q1 + c) : 0u;
      qf[i][2] = in ? *reinterpret_cast<const uint32_t*>(q0 + c + 8) : 0u;
      qf[i][3] = in ? *reinterpret_cast<const uint32_t*>(q1 + c + 8) : 0u;
    }
  }
  float o[VP][2][4];
#pragma unroll
  for (int v = 0; v < VP; ++v)
#pragma unroll
    for (int n = 0; n < 2; ++n) o[v][n][0] = o[v][n][1] = o[v][n][2] = o[v][n][3] = 0.f;
  float m, l;
  int rpos, rlo;
  {                                                   // the row whose softmax this warp keeps
    const int r = R0 + warp;
    m = -INFINITY; l = 0.f;
    rpos = r < nrows ? a.positions[rs + r / H] : -1;
    rlo = a.window > 0 ? max(0, rpos - a.window + 1) : 0;
  }
  const float scale2 = a.scale * LM_LOG2E;
  // ldmatrix rows: 16 keys x two 8-column halves; of the warp's first step (the next one is two blocks on) and of its first
  // column pair (the next one is four blocks on): the swizzled piece within a block is the same for all of them
  const uint32_t q_off = (kw >> 2) * LM_BLK + (lane & 15) * 128 + ((((kw & 3) * 2 + (lane >> 4)) ^ (lane & 7)) << 4);
  const uint32_t v_off = (warp >> 2) * LM_BLK + (lane & 15) * 128 + ((((warp & 3) * 2 + (lane >> 4)) ^ (lane & 7)) << 4);
  int cur = 0;                                        // the stage that holds the tile's first half
  uint32_t phase = 0;
  bool ok = true;
  for (int kt = t0; kt < t1; ++kt) {
    const int s0 = cur, s1 = cur + 1 == ST ? 0 : cur + 1;
    const uint32_t p0 = phase, p1 = s1 == 0 ? phase ^ 1 : phase;
    cur = s1 + 1 == ST ? 0 : s1 + 1;
    phase = cur < s0 ? phase ^ 1 : phase;
    ok = lm_mbar_wait(full(s0), p0) && ok;            // this tile's two stages have landed
    ok = lm_mbar_wait(full(s1), p1) && ok;
    const uint32_t K[2] = {sK + s0 * stage_bytes, sK + s1 * stage_bytes};
    {
      // this warp's columns of its 32 keys: four independent 16 x 8 products, summed over the warps below
      float sc[4][4];
      const uint32_t Kw = (half ? K[1] : K[0]) + q_off;
#pragma unroll
      for (int n = 0; n < 4; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
#pragma unroll
      for (int i = 0; i < LM_KSW; ++i) {
        const int ks = kw + i * LM_KW;
        if (ks < ksteps) {
#pragma unroll
          for (int g = 0; g < 2; ++g) {
            uint32_t bb[4];                           // keys g * 16 .. + 7: halves 0 and 2; + 8 .. 15: halves 1 and 3
            lm_ldm4(bb, Kw + i * 2 * LM_BLK + g * 16 * 128);
            lm_mma(sc[2 * g], qf[i], bb[0], bb[2]);
            lm_mma(sc[2 * g + 1], qf[i], bb[1], bb[3]);
          }
        }
      }
      float* d0 = Ss + (kw * LM_ROWS + (lane >> 2)) * LM_SLD + half * LM_KH + (lane & 3) * 2;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        *reinterpret_cast<float2*>(d0 + n * 8) = make_float2(sc[n][0], sc[n][1]);
        *reinterpret_cast<float2*>(d0 + 8 * LM_SLD + n * 8) = make_float2(sc[n][2], sc[n][3]);
      }
    }
    lm_sync();
    {
      const int j = lo_min + kt * LM_KT + lane * 2;   // two keys per lane
      {
        const int r = warp;
        float x = 0.f, y = 0.f;
#pragma unroll
        for (int w = 0; w < LM_KW; ++w) {
          const float2 v = *reinterpret_cast<const float2*>(Ss + (w * LM_ROWS + r) * LM_SLD + lane * 2);
          x += v.x; y += v.y;
        }
        x = (j <= rpos && j >= rlo) ? x * scale2 : -INFINITY;
        y = (j + 1 <= rpos && j + 1 >= rlo) ? y * scale2 : -INFINITY;
        const float mn = fmaxf(m, warp_max(fmaxf(x, y)));
        const float base = mn == -INFINITY ? 0.f : mn;      // no key yet: every weight is 0
        const float px = lm_ex2(x - base), py = lm_ex2(y - base), corr = lm_ex2(m - base);
        l = l * corr + warp_sum(px + py);
        m = mn;
        *reinterpret_cast<__nv_bfloat162*>(Ps + r * LM_PLD + lane * 2) = __floats2bfloat162_rn(px, py);
        if (lane == 0) cs[r] = corr;
      }
    }
    lm_sync();
    {
      const float c0 = cs[lane >> 2], c1 = cs[(lane >> 2) + 8];
      uint32_t pf[4][4];
      const uint32_t pa = lm_saddr(Ps + (lane & 15) * LM_PLD + (lane >> 4) * 8);
#pragma unroll
      for (int g = 0; g < 4; ++g) lm_ldm4(pf[g], pa + g * 32);
#pragma unroll
      for (int v = 0; v < VP; ++v) {
        const int pr = warp + v * LM_WARPS;
        if (pr < vpairs) {
#pragma unroll
          for (int n = 0; n < 2; ++n) { o[v][n][0] *= c0; o[v][n][1] *= c0; o[v][n][2] *= c1; o[v][n][3] *= c1; }
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            uint32_t bb[4];
            lm_ldm4t(bb, K[g >> 1] + v_off + v * 4 * LM_BLK + (g & 1) * 16 * 128);
            lm_mma(o[v][0], pf[g], bb[0], bb[1]);
            lm_mma(o[v][1], pf[g], bb[2], bb[3]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) { lm_mbar_arrive(empty(s0)); lm_mbar_arrive(empty(s1)); }
    }
  }
  if (lane == 0) { cs[LM_ROWS + warp] = m; cs[2 * LM_ROWS + warp] = ok ? l : __int_as_float(0x7fffffff); }      // copies that never arrived: not a number
  lm_sync();
  const int64_t grow = (int64_t)rs * H + R0;          // this tile's first row among all (token, head) pairs of the step
  if (a.splits > 1) {
    // partial results to the workspace; the CTA of this row tile that arrives last merges them, splits in ascending order of their keys
    const int64_t rows = (int64_t)a.T * H;
    int* count = reinterpret_cast<int*>(a.workspace) + (int64_t)blockIdx.z * gridDim.x + blockIdx.x;
    float* part = reinterpret_cast<float*>(a.workspace) + LM_COUNTERS;
    float* po = part + ((int64_t)blockIdx.y * rows + grow) * a.kv_rank;
    float* pm = part + (int64_t)a.splits * rows * a.kv_rank;
    if (tid < LM_ROWS && R0 + tid < nrows) {
      float* q = pm + ((int64_t)blockIdx.y * rows + grow + tid) * 2;
      q[0] = cs[LM_ROWS + tid]; q[1] = cs[2 * LM_ROWS + tid];
    }
#pragma unroll
    for (int v = 0; v < VP; ++v) {
      const int pr = warp + v * LM_WARPS;
      if (pr < vpairs) {
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int r = (lane >> 2) + 8 * h;
            if (R0 + r < nrows) *reinterpret_cast<float2*>(po + (int64_t)r * a.kv_rank + pr * 16 + n * 8 + (lane & 3) * 2) = make_float2(o[v][n][2 * h], o[v][n][2 * h + 1]);
          }
      }
    }
    __threadfence();                                  // this CTA's part is visible device-wide before it counts itself
    lm_sync();
    if (tid == 0) reinterpret_cast<int*>(cs)[0] = atomicAdd(count, 1) == a.splits - 1;
    lm_sync();
    if (!reinterpret_cast<int*>(cs)[0]) return;
    __threadfence();
    if (tid == 0) *count = 0;                         // ready for the next launch
    const int r = warp;                               // a warp merges one row
    if (R0 + r >= nrows) return;
    const float sk = a.sinks ? a.sinks[(R0 + r) % H] * LM_LOG2E : -INFINITY;
    float M = sk;
    for (int q = 0; q < a.splits; ++q) M = fmaxf(M, __ldcg(pm + ((int64_t)q * rows + grow + r) * 2));
    float den = a.sinks ? exp2f(sk - M) : 0.f;        // the sink logit joins the denominator: no key, no value
    for (int q = 0; q < a.splits; ++q) {
      const float2 ml = __ldcg(reinterpret_cast<const float2*>(pm + ((int64_t)q * rows + grow + r) * 2));
      if (ml.x != -INFINITY) den = fmaf(exp2f(ml.x - M), ml.y, den);
    }
    const float di = 1.f / den;
    for (int c = lane * 4; c < a.kv_rank; c += 128) {
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int q = 0; q < a.splits; ++q) {
        const float mq = __ldcg(pm + ((int64_t)q * rows + grow + r) * 2);
        if (mq == -INFINITY) continue;                // a part without visible keys
        const float f = exp2f(mq - M);
        const float4 v = __ldcg(reinterpret_cast<const float4*>(part + ((int64_t)q * rows + grow + r) * a.kv_rank + c));
        acc.x = fmaf(f, v.x, acc.x); acc.y = fmaf(f, v.y, acc.y); acc.z = fmaf(f, v.z, acc.z); acc.w = fmaf(f, v.w, acc.w);
      }
      __nv_bfloat162 lo = __floats2bfloat162_rn(acc.x * di, acc.y * di), hi = __floats2bfloat162_rn(acc.z * di, acc.w * di);
      uint2 u; u.x = *reinterpret_cast<uint32_t*>(&lo); u.y = *reinterpret_cast<uint32_t*>(&hi);
      *reinterpret_cast<uint2*>((lm_bf16*)a.out + (grow + r) * a.kv_rank + c) = u;
    }
    return;
  }
  float inv[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int r = (lane >> 2) + 8 * h;
    float mm = cs[LM_ROWS + r], ll = cs[2 * LM_ROWS + r], oc = 1.f;
    if (a.sinks) {                                    // the sink logit joins the denominator: no key, no value
      const float sk = a.sinks[(R0 + r) % H] * LM_LOG2E, mn = fmaxf(mm, sk);
      oc = exp2f(mm - mn);
      ll = ll * oc + exp2f(sk - mn);
    }
    inv[h] = oc / ll;
  }
#pragma unroll
  for (int v = 0; v < VP; ++v) {
    const int pr = warp + v * LM_WARPS;
    if (pr < vpairs) {
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int r = (lane >> 2) + 8 * h;
          if (R0 + r < nrows)
            *reinterpret_cast<__nv_bfloat162*>((lm_bf16*)a.out + (grow + r) * a.kv_rank + pr * 16 + n * 8 + (lane & 3) * 2) =
                __floats2bfloat162_rn(o[v][n][2 * h] * inv[h], o[v][n][2 * h + 1] * inv[h]);
        }
    }
  }
}

template <int VP, int ST>
int lm_launch_st(const LatentMqaArgs& a, cudaStream_t st) {
  const int dim = a.kv_rank + a.rot_part;
  const size_t smem = lm_smem(dim, ST);
  CUtensorMap tm;      // the cache as a matrix of rows; the pool's extent only bounds out-of-range handling, which no row reaches
  if (int rc = make_tmap(&tm, a.cache, (int64_t)1 << 30, dim, std::min(a.block_size, LM_KH))) return rc;
  KGE_CUDA_OK(cudaFuncSetAttribute(latent_mqa_kernel<VP, ST>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  KGE_CUDA_OK(launch_pdl(latent_mqa_kernel<VP, ST>, dim3((a.max_q * a.H + LM_ROWS - 1) / LM_ROWS, a.splits, a.B), dim3(LM_WARPS * 32 + 32), smem, st, tm, a));
  return 0;
}
template <int VP>
int lm_launch(const LatentMqaArgs& a, cudaStream_t st) {
  return lm_smem(a.kv_rank + a.rot_part, 5) <= 227 * 1024 ? lm_launch_st<VP, 5>(a, st) : lm_launch_st<VP, 4>(a, st);
}

}  // namespace

bool latent_mqa_ok(int H, int kv_rank, int rot_part, int block_size) {
  return H > 0 && kv_rank % 16 == 0 && rot_part % 16 == 0 && kv_rank > 0 && kv_rank <= 512 && kv_rank + rot_part <= 16 * LM_KSW * LM_KW && kv_rank + rot_part >= 64 && block_size >= 8 && (block_size & (block_size - 1)) == 0;
}
// parts the key range is cut into: a CTA per SM (their stages fill its shared memory), at least 64 keys each
int latent_mqa_splits(int B, int H, int max_q, int64_t keys) {
  const int64_t tiles = (int64_t)B * ((max_q * H + LM_ROWS - 1) / LM_ROWS);
  const int64_t want = 148 / std::max<int64_t>(tiles, 1), most = keys / LM_KT;
  return (int)std::max<int64_t>(1, std::min<int64_t>(std::min(want, most), 16));
}
int64_t latent_mqa_workspace(int T, int H, int kv_rank, int splits) { return splits > 1 ? LM_COUNTERS * 4 + (int64_t)splits * T * H * (kv_rank + 2) * 4 : 0; }

int latent_mqa(const LatentMqaArgs& a, cudaStream_t st) {
  if (a.B <= 0) return 0;
  KGE_REQUIRE(latent_mqa_ok(a.H, a.kv_rank, a.rot_part, a.block_size) && a.B <= 65535 && a.splits >= 1, "latent_mqa: %d heads over rows of %d + %d", a.H, a.kv_rank, a.rot_part);
  KGE_REQUIRE(a.splits == 1 || (a.max_q == 1 && a.workspace && a.workspace_bytes >= latent_mqa_workspace(a.T, a.H, a.kv_rank, a.splits)), "latent_mqa: %d parts need one row per request and a workspace", a.splits);
  KGE_REQUIRE(a.splits == 1 || (int64_t)a.B * ((a.H + LM_ROWS - 1) / LM_ROWS) <= LM_COUNTERS, "latent_mqa: %d parts of too many row tiles", a.splits);
  KGE_REQUIRE(((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.cache) | reinterpret_cast<uintptr_t>(a.out)) & 15) == 0, "latent_mqa: rows must be 16-byte aligned");
  const int pairs = (a.kv_rank / 16 + LM_WARPS - 1) / LM_WARPS;
  return pairs <= 1 ? lm_launch<1>(a, st) : lm_launch<2>(a, st);
}

}  // namespace kge

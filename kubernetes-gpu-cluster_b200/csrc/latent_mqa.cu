// Attention of all query heads of a request over its cached latent rows: every head's query has already been multiplied by
// the head's key up-projection, so one row [c | turned key part] per token serves all heads as key (the whole row) and as
// value (its c part), and a row is read once per 16 (token, head) pairs instead of once per head.
// A CTA of four warps owns 16 query rows - consecutive (token, head) pairs of one request - and walks its part of the
// visible keys in tiles of 32, staged in shared memory by cp.async one tile ahead:
//   S = Q K^T   mma.sync m16n8k16, each warp 8 keys over all kv_rank + rot_part columns, fp32 scores to shared memory
//   softmax     four rows per warp, one key per lane: window mask, running maximum and sum in fp32, P in bfloat16
//   O += P C    each warp its share of the kv_rank columns, fp32 accumulators in registers
// Decode steps split the key range over several CTAs (too few requests to fill the GPU otherwise); a second kernel merges
// their (m, l, O) and adds the sink's share of the denominator.  HBM-bound: a row's bytes are used for 2 * 16 heads' flops.
#include <algorithm>

#include "common.cuh"
#include "hybrid_ops.h"

namespace kge {

namespace {

constexpr int LM_WARPS = 4, LM_KT = 32, LM_ROWS = 16, LM_PAD = 8;
constexpr float LM_LOG2E = 1.4426950408889634f;
typedef __nv_bfloat16 lm_bf16;

__device__ __forceinline__ uint32_t lm_saddr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void lm_cp16(uint32_t dst, const void* src, bool valid) {
  const int sz = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(sz));
}
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

constexpr int LM_SLD = LM_KT + 4, LM_PLD = LM_KT + 8;
size_t lm_smem(int dim) {
  return (size_t)(LM_ROWS + 2 * LM_KT) * (dim + LM_PAD) * 2 + (size_t)LM_ROWS * LM_SLD * 4 + (size_t)LM_ROWS * LM_PLD * 2 + 3 * LM_ROWS * 4;
}

// VP: 16-column pairs of the output per warp
template <int VP>
__global__ void __launch_bounds__(LM_WARPS * 32) latent_mqa_kernel(LatentMqaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) unsigned char lm_raw[];
  const int dim = a.kv_rank + a.rot_part, ld = dim + LM_PAD, H = a.H;
  lm_bf16* Qs = reinterpret_cast<lm_bf16*>(lm_raw);
  lm_bf16* Ks = Qs + LM_ROWS * ld;
  float* Ss = reinterpret_cast<float*>(Ks + 2 * LM_KT * ld);
  lm_bf16* Ps = reinterpret_cast<lm_bf16*>(Ss + LM_ROWS * LM_SLD);
  float* cs = reinterpret_cast<float*>(Ps + LM_ROWS * LM_PLD);      // [16] correction of this tile, then [16] m, [16] l
  const int b = a.req0 + blockIdx.z, rs = a.qsl[b], nrows = (a.qsl[b + 1] - rs) * H, R0 = blockIdx.x * LM_ROWS;
  if (R0 >= nrows) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int pos_first = a.positions[rs + R0 / H], pos_last = a.positions[rs + min(R0 + LM_ROWS - 1, nrows - 1) / H];
  const int lo_min = a.window > 0 ? max(0, pos_first - a.window + 1) : 0;
  const int ntiles = (pos_last - lo_min) / LM_KT + 1, per = (ntiles + a.splits - 1) / a.splits;
  const int t0 = blockIdx.y * per, t1 = min(ntiles, t0 + per);
  const int chunks = dim >> 3;
  const int32_t* bt = a.block_table + (int64_t)b * a.max_blocks;
  const lm_bf16* cache = (const lm_bf16*)a.cache;
  // Q rows (rows beyond the request's repeat its last one; they are never written)
  const lm_bf16* q = (const lm_bf16*)a.q + (int64_t)rs * H * dim;
  for (int i = tid; i < LM_ROWS * chunks; i += LM_WARPS * 32) {
    const int r = i / chunks, c = i % chunks;
    lm_cp16(lm_saddr(Qs + r * ld + c * 8), q + (int64_t)min(R0 + r, nrows - 1) * dim + c * 8, true);
  }
  // a warp stages 8 of a tile's 32 rows; the first eight lanes look up where they live
  auto stage = [&](int kt) {
    lm_bf16* dst = Ks + (kt & 1) * LM_KT * ld + warp * 8 * ld;
    const int j = lo_min + kt * LM_KT + warp * 8 + (lane & 7);
    const int jc = min(j, pos_last);
    const int64_t row = (int64_t)bt[jc / a.block_size] * a.block_size + jc % a.block_size;
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      const int64_t rr = __shfl_sync(0xffffffffu, row, r);
      const bool ok = lo_min + kt * LM_KT + warp * 8 + r <= pos_last;
      const lm_bf16* src = cache + rr * dim;
      for (int c = lane; c < chunks; c += 32) lm_cp16(lm_saddr(dst + r * ld + c * 8), src + c * 8, ok);
    }
  };
  if (t0 < t1) stage(t0);
  asm volatile("cp.async.commit_group;");
  float o[VP][2][4];
#pragma unroll
  for (int v = 0; v < VP; ++v)
#pragma unroll
    for (int n = 0; n < 2; ++n) o[v][n][0] = o[v][n][1] = o[v][n][2] = o[v][n][3] = 0.f;
  float m[4], l[4];
  int rpos[4], rlo[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {                       // the rows whose softmax this warp keeps
    const int r = R0 + warp * 4 + i;
    m[i] = -INFINITY; l[i] = 0.f;
    rpos[i] = r < nrows ? a.positions[rs + r / H] : -1;
    rlo[i] = a.window > 0 ? max(0, rpos[i] - a.window + 1) : 0;
  }
  const float scale2 = a.scale * LM_LOG2E;
  const int ksteps = dim >> 4, vpairs = a.kv_rank >> 4;
  for (int kt = t0; kt < t1; ++kt) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                  // this tile has landed; the other stage's readers are done
    if (kt + 1 < t1) stage(kt + 1);
    asm volatile("cp.async.commit_group;");
    const lm_bf16* K = Ks + (kt & 1) * LM_KT * ld;
    {
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t qa = lm_saddr(Qs + (lane & 15) * ld + (lane >> 4) * 8);
      const lm_bf16* kr = K + (warp * 8 + (lane & 7)) * ld;
      int ks = 0;
#pragma unroll 4
      for (; ks + 1 < ksteps; ks += 2) {
        uint32_t a0[4], a1[4], bb[4];
        lm_ldm4(a0, qa + ks * 32);
        lm_ldm4(a1, qa + ks * 32 + 32);
        lm_ldm4(bb, lm_saddr(kr + ks * 16 + (lane >> 3) * 8));
        lm_mma(s0, a0, bb[0], bb[1]);
        lm_mma(s1, a1, bb[2], bb[3]);
      }
      if (ks < ksteps) {
        uint32_t a0[4], bb[4];
        lm_ldm4(a0, qa + ks * 32);
        lm_ldm4(bb, lm_saddr(kr + ks * 16 + ((lane >> 3) & 1) * 8));
        lm_mma(s0, a0, bb[0], bb[1]);
      }
      float* d0 = Ss + (lane >> 2) * LM_SLD + warp * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(d0) = make_float2((s0[0] + s1[0]) * scale2, (s0[1] + s1[1]) * scale2);
      *reinterpret_cast<float2*>(d0 + 8 * LM_SLD) = make_float2((s0[2] + s1[2]) * scale2, (s0[3] + s1[3]) * scale2);
    }
    __syncthreads();
    {
      const int j = lo_min + kt * LM_KT + lane;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = warp * 4 + i;
        const float s = (j <= rpos[i] && j >= rlo[i]) ? Ss[r * LM_SLD + lane] : -INFINITY;
        const float mn = fmaxf(m[i], warp_max(s));
        const float p = s == -INFINITY ? 0.f : exp2f(s - mn);
        const float corr = mn == -INFINITY ? 1.f : exp2f(m[i] - mn);
        l[i] = l[i] * corr + warp_sum(p);
        m[i] = mn;
        Ps[r * LM_PLD + lane] = __float2bfloat16_rn(p);
        if (lane == 0) cs[r] = corr;
      }
    }
    __syncthreads();
    {
      const float c0 = cs[lane >> 2], c1 = cs[(lane >> 2) + 8];
      uint32_t p0[4], p1[4];
      const uint32_t pa = lm_saddr(Ps + (lane & 15) * LM_PLD + (lane >> 4) * 8);
      lm_ldm4(p0, pa);
      lm_ldm4(p1, pa + 32);
#pragma unroll
      for (int v = 0; v < VP; ++v) {
        const int pr = warp + v * LM_WARPS;
        if (pr < vpairs) {
#pragma unroll
          for (int n = 0; n < 2; ++n) { o[v][n][0] *= c0; o[v][n][1] *= c0; o[v][n][2] *= c1; o[v][n][3] *= c1; }
          uint32_t b0[4], b1[4];
          const uint32_t va = lm_saddr(K + (lane & 15) * ld + pr * 16 + (lane >> 4) * 8);
          lm_ldm4t(b0, va);
          lm_ldm4t(b1, va + 16 * ld * 2);
          lm_mma(o[v][0], p0, b0[0], b0[1]);
          lm_mma(o[v][1], p0, b0[2], b0[3]);
          lm_mma(o[v][0], p1, b1[0], b1[1]);
          lm_mma(o[v][1], p1, b1[2], b1[3]);
        }
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int i = 0; i < 4; ++i) if (lane == 0) { cs[LM_ROWS + warp * 4 + i] = m[i]; cs[2 * LM_ROWS + warp * 4 + i] = l[i]; }
  __syncthreads();
  const int64_t grow = (int64_t)rs * H + R0;          // this tile's first row among all (token, head) pairs of the step
  if (a.splits > 1) {
    float* po = (float*)a.workspace + ((int64_t)blockIdx.y * a.T * H + grow) * a.kv_rank;
    float* pm = (float*)a.workspace + (int64_t)a.splits * a.T * H * a.kv_rank + ((int64_t)blockIdx.y * a.T * H + grow) * 2;
    if (tid < LM_ROWS && R0 + tid < nrows) { pm[tid * 2] = cs[LM_ROWS + tid]; pm[tid * 2 + 1] = cs[2 * LM_ROWS + tid]; }
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

// one block per (token, head): the splits' partial results in ascending order of their keys
__global__ void __launch_bounds__(128) latent_mqa_merge_kernel(LatentMqaArgs a, int64_t row0) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = row0 + blockIdx.x, rows = (int64_t)a.T * a.H;
  const float* pm = (const float*)a.workspace + (int64_t)a.splits * rows * a.kv_rank + row * 2;
  float M = a.sinks ? a.sinks[row % a.H] * LM_LOG2E : -INFINITY;
  const float sk = M;
  for (int s = 0; s < a.splits; ++s) M = fmaxf(M, pm[(int64_t)s * rows * 2]);
  float den = a.sinks ? exp2f(sk - M) : 0.f;
  for (int s = 0; s < a.splits; ++s) {
    const float ms = pm[(int64_t)s * rows * 2];
    if (ms != -INFINITY) den = fmaf(exp2f(ms - M), pm[(int64_t)s * rows * 2 + 1], den);
  }
  const float inv = 1.f / den;
  for (int c = threadIdx.x * 4; c < a.kv_rank; c += 512) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < a.splits; ++s) {
      const float ms = pm[(int64_t)s * rows * 2];
      if (ms == -INFINITY) continue;                  // a part without visible keys
      const float f = exp2f(ms - M);
      const float4 v = *reinterpret_cast<const float4*>((const float*)a.workspace + ((int64_t)s * rows + row) * a.kv_rank + c);
      acc.x = fmaf(f, v.x, acc.x); acc.y = fmaf(f, v.y, acc.y); acc.z = fmaf(f, v.z, acc.z); acc.w = fmaf(f, v.w, acc.w);
    }
    __nv_bfloat162 lo = __floats2bfloat162_rn(acc.x * inv, acc.y * inv), hi = __floats2bfloat162_rn(acc.z * inv, acc.w * inv);
    uint2 u; u.x = *reinterpret_cast<uint32_t*>(&lo); u.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>((lm_bf16*)a.out + row * a.kv_rank + c) = u;
  }
}

template <int VP>
int lm_launch(const LatentMqaArgs& a, cudaStream_t st) {
  const size_t smem = lm_smem(a.kv_rank + a.rot_part);
  KGE_CUDA_OK(cudaFuncSetAttribute(latent_mqa_kernel<VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  KGE_CUDA_OK(launch_pdl(latent_mqa_kernel<VP>, dim3((a.max_q * a.H + LM_ROWS - 1) / LM_ROWS, a.splits, a.B), dim3(LM_WARPS * 32), smem, st, a));
  return 0;
}

}  // namespace

bool latent_mqa_ok(int H, int kv_rank, int rot_part, int block_size) {
  return H > 0 && kv_rank % 16 == 0 && rot_part % 16 == 0 && kv_rank > 0 && kv_rank <= 512 && kv_rank + rot_part <= 640 && block_size > 0;
}
// parts the key range is cut into: enough CTAs for two per SM, at least two tiles of keys each
int latent_mqa_splits(int B, int H, int max_q, int64_t keys) {
  const int64_t tiles = (int64_t)B * ((max_q * H + LM_ROWS - 1) / LM_ROWS);
  const int64_t want = 296 / std::max<int64_t>(tiles, 1), most = keys / (2 * LM_KT);
  return (int)std::max<int64_t>(1, std::min<int64_t>(std::min(want, most), 16));
}
int64_t latent_mqa_workspace(int T, int H, int kv_rank, int splits) { return splits > 1 ? (int64_t)splits * T * H * (kv_rank + 2) * 4 : 0; }

int latent_mqa(const LatentMqaArgs& a, cudaStream_t st) {
  if (a.B <= 0) return 0;
  KGE_REQUIRE(latent_mqa_ok(a.H, a.kv_rank, a.rot_part, a.block_size) && a.B <= 65535 && a.splits >= 1, "latent_mqa: %d heads over rows of %d + %d", a.H, a.kv_rank, a.rot_part);
  KGE_REQUIRE(a.splits == 1 || (a.max_q == 1 && a.workspace && a.workspace_bytes >= latent_mqa_workspace(a.T, a.H, a.kv_rank, a.splits)), "latent_mqa: %d parts need one row per request and a workspace", a.splits);
  KGE_REQUIRE(((reinterpret_cast<uintptr_t>(a.q) | reinterpret_cast<uintptr_t>(a.cache) | reinterpret_cast<uintptr_t>(a.out)) & 15) == 0, "latent_mqa: rows must be 16-byte aligned");
  const int pairs = (a.kv_rank / 16 + LM_WARPS - 1) / LM_WARPS;
  if (int rc = pairs <= 2 ? lm_launch<2>(a, st) : pairs <= 4 ? lm_launch<4>(a, st) : lm_launch<8>(a, st)) return rc;
  // one row per request: the requests' rows follow one another from the first request's on
  if (a.splits > 1) KGE_CUDA_OK(launch_pdl(latent_mqa_merge_kernel, dim3((unsigned)(a.B * a.H)), dim3(128), 0, st, a, (int64_t)a.req0 * a.H));
  return 0;
}

}  // namespace kge

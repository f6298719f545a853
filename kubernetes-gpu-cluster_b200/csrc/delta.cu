// Gated delta rule for layer-list models: each head carries a dim x vdim matrix S in fp32 that decays per key channel and
// per token and is corrected towards the token's value along its key,
//     S <- diag(g_t) S;   u = b_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t.
// A value column of S depends on its own entries only, so columns are spread over threads, warps and blocks: a thread owns
// CPT neighbouring columns of KPT of the key channels, KQ neighbouring lanes together hold all channels and sum the two
// read-outs (along k and along q) by shuffles, and o_t follows from the decayed state without waiting for its update,
//     o_t = S'^T q_t + (k_t . q_t) u,    S' = diag(g_t) S.
// The rows' operands are staged CT tokens at a time with cp.async, one stage ahead, for all warps of the block; inside a
// stage the warps run without a barrier.  S lives in the request's state slot between steps, so a prompt cut anywhere
// continues exactly.
#include <algorithm>

#include "common.cuh"
#include "elt_access.cuh"
#include "f32x2.cuh"
#include "hybrid_ops.h"

namespace kge {

namespace {

__device__ __forceinline__ void dl_cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void dl_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
template <int N> __device__ __forceinline__ void dl_ld(const float* p, float (&v)[N]) {
  if constexpr (N == 4) ld4(p, v);
  else { const float2 t = *reinterpret_cast<const float2*>(p); v[0] = t.x; v[1] = t.y; }
}
template <int N> __device__ __forceinline__ void dl_st(float* p, const float (&v)[N]) {
  if constexpr (N == 4) st4(p, v);
  else *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
}
// a packed pair holds two neighbouring key channels of one column

// KQ lanes x KPT channels cover dim; CPT columns per thread; a block owns `cols` value columns from blockIdx.x * cols on.
// VEC: operand rows in 16-byte pieces, state rows and outputs in pieces of CPT columns.
template <int KQ, int KPT, int CPT, int CT, bool VEC>
__global__ void __launch_bounds__(256) delta_scan_kernel(DeltaArgs a, int cols) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int DK = KQ * KPT, NP = KPT / 2;
  extern __shared__ __align__(16) float dl_sm[];
  const int vld = (cols + 3) & ~3, per_tok = 3 * DK + vld;
  float* beta_s = dl_sm + 2 * CT * per_tok;          // [2][CT]
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, nt = blockDim.x, lane = tid & 31;
  const int r0 = a.qsl[b], r1 = a.qsl[b + 1];
  if (r0 >= r1) return;
  const int dim = a.dim, vdim = a.vdim, hk = h / (a.H / a.G), HD = a.H * dim, HV = a.H * vdim;
  const int c0 = blockIdx.x * cols, nc = min(cols, vdim - c0);
  const int kq = tid % KQ, col = (tid / KQ) * CPT;   // this thread's channel slice and first column (within the block)
  const bool fresh = a.positions[r0] == 0;
  float* Sg = a.state + (int64_t)a.slots[b] * a.slot_stride + (int64_t)h * dim * vdim + c0;
  // channels of pair i: chunk i / 2 of four channels, the KQ lanes' chunks side by side
  auto chan = [&](int i) { return ((i >> 1) * KQ + kq) * 4 + (i & 1) * 2; };
  f2 S[NP][CPT];
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    float x[2][CPT] = {};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = chan(i) + e;
      if (!fresh && k < dim) {
        if (VEC) { if (col < nc) dl_ld<CPT>(Sg + (int64_t)k * vdim + col, x[e]); }
        else {
#pragma unroll
          for (int j = 0; j < CPT; ++j) if (col + j < nc) x[e][j] = Sg[(int64_t)k * vdim + col + j];
        }
      }
    }
#pragma unroll
    for (int j = 0; j < CPT; ++j) S[i][j] = pk(x[0][j], x[1][j]);
  }
  if (dim < DK || nc < vld) {                        // channels and columns that are never staged stay zero
    for (int i = tid; i < 2 * CT * per_tok; i += nt) dl_sm[i] = 0.f;
    __syncthreads();
  }
  const float* src[4] = {a.qkv + (int64_t)(a.G + hk) * dim, a.qkv + (int64_t)hk * dim, a.decay + (int64_t)h * dim, a.qkv + (int64_t)2 * a.G * dim + (int64_t)h * vdim + c0};
  constexpr int W = VEC ? 4 : 1;
  const int piece_k = dim / W, roles = 3 * piece_k + nc / W;                    // pieces of a token's k, q, decay and value columns
  const int tpar = max(1, nt / roles), role0 = nt >= roles ? tid % roles : tid, role_step = nt >= roles ? roles : nt;
  const int tok0 = nt >= roles ? (tid / roles < tpar ? tid / roles : CT) : 0;  // left-over threads copy nothing
  auto beta_raw = [&](int t) -> float {
    if (t >= r1) return 0.f;
    const int64_t o = (int64_t)t * a.ldb + h;
    return a.elt == KGE_ELT_F32 ? ((const float*)a.beta_pre)[o] : __bfloat162float(((const __nv_bfloat16*)a.beta_pre)[o]);
  };
  float braw = tid < CT ? beta_raw(r0 + tid) : 0.f;  // the raw step size is requested a stage before it is used
  auto stage = [&](int t0, int s) {
    float* base = dl_sm + s * CT * per_tok;
    const int n = min(CT, r1 - t0);
    // a thread copies one piece (16 bytes, or one number) of an operand for every `tpar`-th token of the stage
    for (int r = role0; r < roles; r += role_step) {
      const int op = r < piece_k ? 0 : r < 2 * piece_k ? 1 : r < 3 * piece_k ? 2 : 3, c = (r - op * piece_k) * W;
      const int64_t step = op == 2 ? HD : a.ld;
      const float* p = (op == 0 ? src[0] : op == 1 ? src[1] : op == 2 ? src[2] : src[3]) + (int64_t)(t0 + tok0) * step + c;
      float* d = base + tok0 * per_tok + op * DK + c;
      for (int t = tok0; t < n; t += tpar, p += step * tpar, d += per_tok * tpar) { if (VEC) dl_cp16(d, p); else dl_cp4(d, p); }
    }
    if (tid < CT) {
      beta_s[s * CT + tid] = 1.f / (1.f + expf(-braw));
      braw = beta_raw(t0 + CT + tid);
    }
    asm volatile("cp.async.commit_group;");
  };
  stage(r0, 0);
  int s = 0;
  for (int t0 = r0; t0 < r1; t0 += CT, s ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                 // the stage has landed; the other one's readers are done
    if (t0 + CT < r1) stage(t0 + CT, s ^ 1);
    const int n = min(CT, r1 - t0);
    const float* d = dl_sm + s * CT * per_tok;
    float* op = a.o32 + (int64_t)t0 * HV + (int64_t)h * vdim + c0 + col;
    for (int t = 0; t < n; ++t, d += per_tok, op += HV) {
      f2 k[NP], dk2[CPT], dq2[CPT], kq2 = 0ull;
#pragma unroll
      for (int j = 0; j < CPT; ++j) dk2[j] = dq2[j] = 0ull;
#pragma unroll
      for (int c = 0; c < KPT / 4; ++c) {
        const int o = (c * KQ + kq) * 4;
        const ulonglong2 kk = *reinterpret_cast<const ulonglong2*>(d + o), qq = *reinterpret_cast<const ulonglong2*>(d + DK + o), gg = *reinterpret_cast<const ulonglong2*>(d + 2 * DK + o);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = c * 2 + e;
          const f2 ke = e ? kk.y : kk.x, qe = e ? qq.y : qq.x, ge = e ? gg.y : gg.x;
          k[i] = ke;
          kq2 = fma2(ke, qe, kq2);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            const f2 x = mul2(S[i][j], ge);
            S[i][j] = x;
            dk2[j] = fma2(x, ke, dk2[j]);
            dq2[j] = fma2(x, qe, dq2[j]);
          }
        }
      }
      const float be = beta_s[s * CT + t];
      float v[CPT], u[CPT], dk[CPT], dq[CPT], kq_dot = sum2(kq2);
      dl_ld<CPT>(d + 3 * DK + col, v);
#pragma unroll
      for (int j = 0; j < CPT; ++j) { dk[j] = sum2(dk2[j]); dq[j] = sum2(dq2[j]); }
#pragma unroll
      for (int off = 1; off < KQ; off <<= 1) kq_dot += __shfl_xor_sync(0xffffffffu, kq_dot, off);
      if constexpr (CPT == 2) {
        // four sums over the KQ lanes: two exchanges split them (see below)
        const bool b0 = kq & 1, b1 = kq & 2;
        const float x0 = (b0 ? dq[0] : dk[0]) + __shfl_xor_sync(0xffffffffu, b0 ? dk[0] : dq[0], 1);
        const float x1 = (b0 ? dq[1] : dk[1]) + __shfl_xor_sync(0xffffffffu, b0 ? dk[1] : dq[1], 1);
        float y = (b1 ? x1 : x0) + __shfl_xor_sync(0xffffffffu, b1 ? x0 : x1, 2);
#pragma unroll
        for (int off = 4; off < KQ; off <<= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
        const int g0 = lane & ~(KQ - 1);
        u[0] = be * (v[0] - __shfl_sync(0xffffffffu, y, g0));
        u[1] = be * (v[1] - __shfl_sync(0xffffffffu, y, g0 + 2));
        if (b0 && kq < 4) { const int j = b1 ? 1 : 0; if (col + j < nc) op[j] = fmaf(kq_dot, b1 ? u[1] : u[0], y); }
      } else if constexpr (KQ >= 8) {
        // eight sums over the KQ lanes: three exchanges split them, so each lane ends with one; then every lane fetches the
        // four sums along k, and the lanes that hold a sum along q write its output
        const bool b0 = kq & 1, b1 = kq & 2, b2 = kq & 4;
        float x[4], z[2];
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] = (b0 ? dq[j] : dk[j]) + __shfl_xor_sync(0xffffffffu, b0 ? dk[j] : dq[j], 1);
#pragma unroll
        for (int j = 0; j < 2; ++j) z[j] = (b1 ? x[2 + j] : x[j]) + __shfl_xor_sync(0xffffffffu, b1 ? x[j] : x[2 + j], 2);
        float y = (b2 ? z[1] : z[0]) + __shfl_xor_sync(0xffffffffu, b2 ? z[0] : z[1], 4);
        
#pragma unroll
        for (int off = 8; off < KQ; off <<= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
        const int g0 = lane & ~(KQ - 1);
#pragma unroll
        for (int j = 0; j < 4; ++j) u[j] = be * (v[j] - __shfl_sync(0xffffffffu, y, g0 + (j >> 1) * 2 + (j & 1) * 4));
        if (b0 && kq < 8) {
          const int j = (b1 ? 2 : 0) + (b2 ? 1 : 0);
          const float uj = b1 ? (b2 ? u[3] : u[2]) : (b2 ? u[1] : u[0]);
          if (col + j < nc) op[j] = fmaf(kq_dot, uj, y);
        }
      } else {
#pragma unroll
        for (int off = KQ / 2; off > 0; off >>= 1)
#pragma unroll
          for (int j = 0; j < CPT; ++j) { dk[j] += __shfl_xor_sync(0xffffffffu, dk[j], off); dq[j] += __shfl_xor_sync(0xffffffffu, dq[j], off); }
#pragma unroll
        for (int j = 0; j < CPT; ++j) { u[j] = be * (v[j] - dk[j]); dq[j] = fmaf(kq_dot, u[j], dq[j]); }
        if (kq == 0 && col < nc) {
          if (VEC) dl_st<CPT>(op, dq);
          else {
#pragma unroll
            for (int j = 0; j < CPT; ++j) if (col + j < nc) op[j] = dq[j];
          }
        }
      }
      f2 uu[CPT];
#pragma unroll
      for (int j = 0; j < CPT; ++j) uu[j] = pk(u[j], u[j]);
#pragma unroll
      for (int i = 0; i < NP; ++i)
#pragma unroll
        for (int j = 0; j < CPT; ++j) S[i][j] = fma2(k[i], uu[j], S[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    float x[2][CPT];
#pragma unroll
    for (int j = 0; j < CPT; ++j) upk(S[i][j], x[0][j], x[1][j]);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int k = chan(i) + e;
      if (k < dim) {
        if (VEC) { if (col < nc) dl_st<CPT>(Sg + (int64_t)k * vdim + col, x[e]); }
        else {
#pragma unroll
          for (int j = 0; j < CPT; ++j) if (col + j < nc) Sg[(int64_t)k * vdim + col + j] = x[e][j];
        }
      }
    }
  }
}

template <int KQ, int KPT, int CPT, int CT>
int delta_launch(const DeltaArgs& a, bool vec, cudaStream_t st) {
  // up to eight warps per block (four in one-token steps); fewer (more blocks) for heads with few columns
  const int warp_cols = 32 / KQ * CPT;
  const int warps = std::min(CT == 1 ? 4 : 8, (a.vdim + warp_cols - 1) / warp_cols), cols = warps * warp_cols;
  const dim3 grid((a.vdim + cols - 1) / cols, a.H, a.B), block(warps * 32);
  const size_t smem = (size_t)(2 * CT * (3 * KQ * KPT + ((cols + 3) & ~3)) + 2 * CT) * 4;
  auto kern = vec ? delta_scan_kernel<KQ, KPT, CPT, CT, true> : delta_scan_kernel<KQ, KPT, CPT, CT, false>;
  if (smem > 48 * 1024) KGE_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  KGE_CUDA_OK(launch_pdl(kern, grid, block, smem, st, a, cols));
  return 0;
}

}  // namespace

int delta_scan(const DeltaArgs& a, cudaStream_t st) {
  if (a.T <= 0) return 0;
  KGE_REQUIRE(a.dim > 0 && a.dim <= 256 && a.vdim > 0 && a.G > 0 && a.H % a.G == 0 && a.H <= 65535 && a.B <= 65535, "delta_scan: %d heads on %d of %d x %d", a.H, a.G, a.dim, a.vdim);
  const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ld % 4 == 0 && a.slot_stride % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.qkv) | reinterpret_cast<uintptr_t>(a.decay) | reinterpret_cast<uintptr_t>(a.o32) | reinterpret_cast<uintptr_t>(a.state)) & 15) == 0;
  if (a.T == a.B) {               // one row per request: one token per stage
    if (a.dim <= 32) return delta_launch<4, 8, 4, 1>(a, vec, st);
    if (a.dim <= 64) return delta_launch<4, 16, 4, 1>(a, vec, st);
    if (a.dim <= 128) return delta_launch<8, 16, 4, 1>(a, vec, st);
    return delta_launch<16, 16, 4, 1>(a, vec, st);
  }
  if (a.dim <= 32) return delta_launch<4, 8, 2, 16>(a, vec, st);
  if (a.dim <= 64) return delta_launch<4, 16, 2, 16>(a, vec, st);
  if (a.dim <= 128) return delta_launch<8, 16, 2, 16>(a, vec, st);
  return delta_launch<16, 16, 2, 8>(a, vec, st);
}

}  // namespace kge

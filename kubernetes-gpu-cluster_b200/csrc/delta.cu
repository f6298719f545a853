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

// KQ lanes x KPT channels cover dim; CPT columns per thread; a block owns `cols` value columns from blockIdx.x * cols on.
// VEC: operand rows in 16-byte pieces, state rows and outputs in pieces of CPT columns.
template <int KQ, int KPT, int CPT, int CT, bool VEC>
__global__ void __launch_bounds__(128) delta_scan_kernel(DeltaArgs a, int cols) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int DK = KQ * KPT;
  extern __shared__ __align__(16) float dl_sm[];
  const int vld = (cols + 3) & ~3, per_tok = 3 * DK + vld;
  float* beta_s = dl_sm + 2 * CT * per_tok;          // [2][CT]
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5, nw = nt >> 5;
  const int r0 = a.qsl[b], r1 = a.qsl[b + 1];
  if (r0 >= r1) return;
  const int dim = a.dim, vdim = a.vdim, hk = h / (a.H / a.G), HD = a.H * dim, HV = a.H * vdim;
  const int c0 = blockIdx.x * cols, nc = min(cols, vdim - c0);
  const int kq = tid % KQ, col = (tid / KQ) * CPT;   // this thread's channel slice and first column (within the block)
  const bool fresh = a.positions[r0] == 0;
  float* Sg = a.state + (int64_t)a.slots[b] * a.slot_stride + (int64_t)h * dim * vdim + c0;
  // channel of register i: chunk i / 4 of four channels, the KQ lanes' chunks side by side
  float S[KPT][CPT];
#pragma unroll
  for (int i = 0; i < KPT; ++i) {
    const int k = ((i >> 2) * KQ + kq) * 4 + (i & 3);
#pragma unroll
    for (int j = 0; j < CPT; ++j) S[i][j] = 0.f;
    if (!fresh && k < dim) {
      if (VEC) { if (col < nc) dl_ld<CPT>(Sg + (int64_t)k * vdim + col, S[i]); }
      else {
#pragma unroll
        for (int j = 0; j < CPT; ++j) if (col + j < nc) S[i][j] = Sg[(int64_t)k * vdim + col + j];
      }
    }
  }
  if (dim < DK || nc < vld) {                        // channels and columns that are never staged stay zero
    for (int i = tid; i < 2 * CT * per_tok; i += nt) dl_sm[i] = 0.f;
    __syncthreads();
  }
  const float* src[4] = {a.qkv + (int64_t)(a.G + hk) * dim, a.qkv + (int64_t)hk * dim, a.decay + (int64_t)h * dim, a.qkv + (int64_t)2 * a.G * dim + (int64_t)h * vdim + c0};
  auto beta_raw = [&](int t) -> float {
    if (t >= r1) return 0.f;
    const int64_t o = (int64_t)t * a.ldb + h;
    return a.elt == KGE_ELT_F32 ? ((const float*)a.beta_pre)[o] : __bfloat162float(((const __nv_bfloat16*)a.beta_pre)[o]);
  };
  float braw = tid < CT ? beta_raw(r0 + tid) : 0.f;  // the raw step size is requested a stage before it is used
  auto stage = [&](int t0, int s) {
    float* base = dl_sm + s * CT * per_tok;
    const int n = min(CT, r1 - t0);
    for (int it = warp; it < n * 4; it += nw) {      // one warp per (token, operand)
      const int t = it >> 2, op = it & 3;
      const float* p = (op == 0 ? src[0] : op == 1 ? src[1] : op == 2 ? src[2] : src[3]) + (int64_t)(t0 + t) * (op == 2 ? HD : a.ld);
      float* d = base + t * per_tok + op * DK;
      const int w = op == 3 ? nc : dim;
      if (VEC) for (int c = lane * 4; c < w; c += 128) dl_cp16(d + c, p + c);
      else for (int c = lane; c < w; c += 32) dl_cp4(d + c, p + c);
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
      float k[KPT], dk[CPT], dq[CPT], kq_dot = 0.f;
#pragma unroll
      for (int j = 0; j < CPT; ++j) dk[j] = dq[j] = 0.f;
#pragma unroll
      for (int c = 0; c < KPT / 4; ++c) {
        const int o = (c * KQ + kq) * 4;
        float kk[4], qq[4], gg[4];
        ld4(d + o, kk); ld4(d + DK + o, qq); ld4(d + 2 * DK + o, gg);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          k[c * 4 + i] = kk[i];
          kq_dot = fmaf(kk[i], qq[i], kq_dot);
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            const float x = S[c * 4 + i][j] * gg[i];
            S[c * 4 + i][j] = x;
            dk[j] = fmaf(x, kk[i], dk[j]);
            dq[j] = fmaf(x, qq[i], dq[j]);
          }
        }
      }
      const float be = beta_s[s * CT + t];
      float v[CPT], u[CPT];
      dl_ld<CPT>(d + 3 * DK + col, v);
      if constexpr (CPT == 2) {
        // four sums over the KQ lanes: the lanes split them in two exchanges, so each ends with one sum; then every lane
        // fetches the two sums along k, and the lanes that hold a sum along q write its output
        const bool b0 = kq & 1, b1 = kq & 2;
        float x0 = b0 ? dq[0] : dk[0], x1 = b0 ? dq[1] : dk[1];
        x0 += __shfl_xor_sync(0xffffffffu, b0 ? dk[0] : dq[0], 1);
        x1 += __shfl_xor_sync(0xffffffffu, b0 ? dk[1] : dq[1], 1);
        float y = b1 ? x1 : x0;
        y += __shfl_xor_sync(0xffffffffu, b1 ? x0 : x1, 2);
#pragma unroll
        for (int off = 4; off < KQ; off <<= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
#pragma unroll
        for (int off = 1; off < KQ; off <<= 1) kq_dot += __shfl_xor_sync(0xffffffffu, kq_dot, off);
        const int g0 = lane & ~(KQ - 1);
        u[0] = be * (v[0] - __shfl_sync(0xffffffffu, y, g0));
        u[1] = be * (v[1] - __shfl_sync(0xffffffffu, y, g0 + 2));
        if (b0 && kq < 4) {
          const int j = b1 ? 1 : 0;
          if (col + j < nc) op[j] = fmaf(kq_dot, b1 ? u[1] : u[0], y);
        }
      } else {
#pragma unroll
        for (int off = KQ / 2; off > 0; off >>= 1) {
          kq_dot += __shfl_xor_sync(0xffffffffu, kq_dot, off);
#pragma unroll
          for (int j = 0; j < CPT; ++j) { dk[j] += __shfl_xor_sync(0xffffffffu, dk[j], off); dq[j] += __shfl_xor_sync(0xffffffffu, dq[j], off); }
        }
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
#pragma unroll
      for (int i = 0; i < KPT; ++i)
#pragma unroll
        for (int j = 0; j < CPT; ++j) S[i][j] = fmaf(k[i], u[j], S[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < KPT; ++i) {
    const int k = ((i >> 2) * KQ + kq) * 4 + (i & 3);
    if (k < dim) {
      if (VEC) { if (col < nc) dl_st<CPT>(Sg + (int64_t)k * vdim + col, S[i]); }
      else {
#pragma unroll
        for (int j = 0; j < CPT; ++j) if (col + j < nc) Sg[(int64_t)k * vdim + col + j] = S[i][j];
      }
    }
  }
}

template <int KQ, int KPT, int CPT, int CT>
int delta_launch(const DeltaArgs& a, bool vec, cudaStream_t st) {
  // up to four warps per block; fewer (more blocks) for heads with few columns
  const int warp_cols = 32 / KQ * CPT;
  const int warps = std::min(4, (a.vdim + warp_cols - 1) / warp_cols), cols = warps * warp_cols;
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
  if (a.T == a.B) {               // one row per request: the state is the traffic - 16-byte pieces of it, one token per stage
    if (a.dim <= 32) return delta_launch<4, 8, 4, 1>(a, vec, st);
    if (a.dim <= 64) return delta_launch<4, 16, 4, 1>(a, vec, st);
    if (a.dim <= 128) return delta_launch<8, 16, 4, 1>(a, vec, st);
    return delta_launch<16, 16, 4, 1>(a, vec, st);
  }
  if (a.dim <= 32) return delta_launch<4, 8, 2, 8>(a, vec, st);
  if (a.dim <= 64) return delta_launch<4, 16, 2, 8>(a, vec, st);
  if (a.dim <= 128) return delta_launch<8, 16, 2, 8>(a, vec, st);
  return delta_launch<16, 16, 2, 4>(a, vec, st);
}

}  // namespace kge

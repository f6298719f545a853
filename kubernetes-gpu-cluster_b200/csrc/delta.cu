// Gated delta rule for layer-list models: each head carries a dim x vdim matrix S in fp32 that decays per key channel and
// per token and is corrected towards the token's value along its key,
//     S <- diag(g_t) S;   u = b_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t.
// A value column of S depends on its own entries only, so columns are spread over threads and blocks: a thread owns four
// neighbouring columns of KPT of the key channels, KQ neighbouring lanes together hold all of them and sum the two read-outs
// (along k and along q) by shuffles, and o_t follows from the decayed state without waiting for its update,
//     o_t = S'^T q_t + (k_t . q_t) u,    S' = diag(g_t) S.
// The rows' operands are staged several tokens at a time with cp.async, one stage ahead.  S lives in the request's state
// slot between steps, so a prompt cut anywhere continues exactly.
#include <algorithm>

#include "common.cuh"
#include "elt_access.cuh"
#include "hybrid_ops.h"

namespace kge {

namespace {

constexpr int DL_KPT = 16;      // key channels per lane

__device__ __forceinline__ void dl_cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void dl_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

// KQ lanes x DL_KPT channels cover dim; CT tokens per stage; a block owns `cols` value columns from blockIdx.x * cols on.
// VEC: operand rows, state rows and outputs in 16-byte pieces.
template <typename E, int KQ, int CT, bool VEC>
__global__ void __launch_bounds__(256) delta_scan_kernel(DeltaArgs a, int cols) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int DK = KQ * DL_KPT;
  extern __shared__ __align__(16) float dl_sm[];
  const int vld = (cols + 3) & ~3, per_tok = 3 * DK + vld;
  float* beta_s = dl_sm + 2 * CT * per_tok;          // [2][CT]
  const int h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, nt = blockDim.x;
  const int r0 = a.qsl[b], r1 = a.qsl[b + 1];
  if (r0 >= r1) return;
  const int dim = a.dim, vdim = a.vdim, hk = h / (a.H / a.G), HD = a.H * dim, HV = a.H * vdim;
  const int c0 = blockIdx.x * cols, nc = min(cols, vdim - c0);
  const int kq = tid % KQ, col = (tid / KQ) * 4;     // this thread's channel slice and first column (within the block)
  const bool fresh = a.positions[r0] == 0;
  float* Sg = a.state + (int64_t)a.slots[b] * a.slot_stride + (int64_t)h * dim * vdim + c0;
  // channel k of register i: chunk (i / 4) of four channels, KQ chunks side by side
  float S[DL_KPT][4];
#pragma unroll
  for (int i = 0; i < DL_KPT; ++i) {
    const int k = ((i >> 2) * KQ + kq) * 4 + (i & 3);
#pragma unroll
    for (int j = 0; j < 4; ++j) S[i][j] = 0.f;
    if (!fresh && k < dim) {
      if (VEC) { if (col < nc) ld4(Sg + (int64_t)k * vdim + col, S[i]); }
      else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (col + j < nc) S[i][j] = Sg[(int64_t)k * vdim + col + j];
      }
    }
  }
  if (dim < DK || nc < vld) {                        // channels and columns that are never staged stay zero
    for (int i = tid; i < 2 * CT * per_tok; i += nt) dl_sm[i] = 0.f;
    __syncthreads();
  }
  const float* qp = a.qkv + (int64_t)hk * dim;
  const float* kp = a.qkv + (int64_t)(a.G + hk) * dim;
  const float* vp = a.qkv + (int64_t)2 * a.G * dim + (int64_t)h * vdim + c0;
  const float* gp = a.decay + (int64_t)h * dim;
  auto stage = [&](int t0, int s) {
    float* base = dl_sm + s * CT * per_tok;
    const int n = min(CT, r1 - t0);
    if (VEC) {
      const int kc = dim >> 2, vc = (nc + 3) >> 2, per = 3 * kc + vc;
      for (int i = tid; i < n * per; i += nt) {
        const int t = i / per, u = i % per;
        const int64_t row = t0 + t;
        float* d = base + t * per_tok;
        if (u < kc) dl_cp16(d + u * 4, kp + row * a.ld + u * 4);
        else if (u < 2 * kc) dl_cp16(d + DK + (u - kc) * 4, qp + row * a.ld + (u - kc) * 4);
        else if (u < 3 * kc) dl_cp16(d + 2 * DK + (u - 2 * kc) * 4, gp + row * HD + (u - 2 * kc) * 4);
        else dl_cp16(d + 3 * DK + (u - 3 * kc) * 4, vp + row * a.ld + (u - 3 * kc) * 4);
      }
    } else {
      const int per = 3 * dim + nc;
      for (int i = tid; i < n * per; i += nt) {
        const int t = i / per, u = i % per;
        const int64_t row = t0 + t;
        float* d = base + t * per_tok;
        if (u < dim) dl_cp4(d + u, kp + row * a.ld + u);
        else if (u < 2 * dim) dl_cp4(d + DK + (u - dim), qp + row * a.ld + (u - dim));
        else if (u < 3 * dim) dl_cp4(d + 2 * DK + (u - 2 * dim), gp + row * HD + (u - 2 * dim));
        else dl_cp4(d + 3 * DK + (u - 3 * dim), vp + row * a.ld + (u - 3 * dim));
      }
    }
    for (int t = tid; t < n; t += nt) beta_s[s * CT + t] = 1.f / (1.f + expf(-ldf((const E*)a.beta_pre + (int64_t)(t0 + t) * a.ldb + h)));
    asm volatile("cp.async.commit_group;");
  };
  stage(r0, 0);
  int s = 0;
  for (int t0 = r0; t0 < r1; t0 += CT, s ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                 // the stage has landed; the other one's readers are done
    if (t0 + CT < r1) stage(t0 + CT, s ^ 1);
    const int n = min(CT, r1 - t0);
    for (int t = 0; t < n; ++t) {
      const float* d = dl_sm + (s * CT + t) * per_tok;
      float k[DL_KPT], dk[4] = {0.f, 0.f, 0.f, 0.f}, dq[4] = {0.f, 0.f, 0.f, 0.f}, kq_dot = 0.f;
#pragma unroll
      for (int c = 0; c < DL_KPT / 4; ++c) {
        const int o = (c * KQ + kq) * 4;
        const float4 k4 = *reinterpret_cast<const float4*>(d + o), q4 = *reinterpret_cast<const float4*>(d + DK + o), g4 = *reinterpret_cast<const float4*>(d + 2 * DK + o);
        const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w}, gg[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          k[c * 4 + i] = kk[i];
          kq_dot = fmaf(kk[i], qq[i], kq_dot);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float x = S[c * 4 + i][j] * gg[i];
            S[c * 4 + i][j] = x;
            dk[j] = fmaf(x, kk[i], dk[j]);
            dq[j] = fmaf(x, qq[i], dq[j]);
          }
        }
      }
#pragma unroll
      for (int off = KQ / 2; off > 0; off >>= 1) {
        kq_dot += __shfl_xor_sync(0xffffffffu, kq_dot, off);
#pragma unroll
        for (int j = 0; j < 4; ++j) { dk[j] += __shfl_xor_sync(0xffffffffu, dk[j], off); dq[j] += __shfl_xor_sync(0xffffffffu, dq[j], off); }
      }
      const float be = beta_s[s * CT + t];
      float v[4] = {0.f, 0.f, 0.f, 0.f}, u[4], o[4];
      if (col < vld) { const float4 v4 = *reinterpret_cast<const float4*>(d + 3 * DK + col); v[0] = v4.x; v[1] = v4.y; v[2] = v4.z; v[3] = v4.w; }
#pragma unroll
      for (int j = 0; j < 4; ++j) { u[j] = be * (v[j] - dk[j]); o[j] = fmaf(kq_dot, u[j], dq[j]); }
#pragma unroll
      for (int i = 0; i < DL_KPT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) S[i][j] = fmaf(k[i], u[j], S[i][j]);
      if (kq == 0 && col < nc) {
        float* op = a.o32 + (int64_t)(t0 + t) * HV + (int64_t)h * vdim + c0 + col;
        if (VEC) st4(op, o);
        else {
#pragma unroll
          for (int j = 0; j < 4; ++j) if (col + j < nc) op[j] = o[j];
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < DL_KPT; ++i) {
    const int k = ((i >> 2) * KQ + kq) * 4 + (i & 3);
    if (k < dim) {
      if (VEC) { if (col < nc) st4(Sg + (int64_t)k * vdim + col, S[i]); }
      else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (col + j < nc) Sg[(int64_t)k * vdim + col + j] = S[i][j];
      }
    }
  }
}

template <typename E, int KQ, int CT>
int delta_launch(const DeltaArgs& a, bool vec, cudaStream_t st) {
  // columns per block: at least a warp's worth; fewer columns (more blocks) while the grid would leave SMs idle
  const int warp_cols = 128 / KQ, most = 256 / KQ * 4;
  int cols = std::min((a.vdim + warp_cols - 1) / warp_cols * warp_cols, most);
  while (cols > warp_cols && (int64_t)a.B * a.H * ((a.vdim + cols - 1) / cols) < 296) cols = std::max(warp_cols, (cols / 2 + warp_cols - 1) / warp_cols * warp_cols);
  const dim3 grid((a.vdim + cols - 1) / cols, a.H, a.B), block(cols / 4 * KQ);
  const size_t smem = (size_t)(2 * CT * (3 * KQ * DL_KPT + ((cols + 3) & ~3)) + 2 * CT) * 4;
  auto kern = vec ? delta_scan_kernel<E, KQ, CT, true> : delta_scan_kernel<E, KQ, CT, false>;
  if (smem > 48 * 1024) KGE_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  KGE_CUDA_OK(launch_pdl(kern, grid, block, smem, st, a, cols));
  return 0;
}

template <typename E>
int delta_scan_t(const DeltaArgs& a, cudaStream_t st) {
  const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ld % 4 == 0 && a.slot_stride % 4 == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.qkv) | reinterpret_cast<uintptr_t>(a.decay) | reinterpret_cast<uintptr_t>(a.o32) | reinterpret_cast<uintptr_t>(a.state)) & 15) == 0;
  if (a.dim <= 32) return delta_launch<E, 2, 8>(a, vec, st);
  if (a.dim <= 64) return delta_launch<E, 4, 8>(a, vec, st);
  if (a.dim <= 128) return delta_launch<E, 8, 8>(a, vec, st);
  return delta_launch<E, 16, 4>(a, vec, st);
}

}  // namespace

int delta_scan(const DeltaArgs& a, cudaStream_t st) {
  if (a.T <= 0) return 0;
  KGE_REQUIRE(a.dim > 0 && a.dim <= 256 && a.vdim > 0 && a.G > 0 && a.H % a.G == 0 && a.H <= 65535 && a.B <= 65535, "delta_scan: %d heads on %d of %d x %d", a.H, a.G, a.dim, a.vdim);
  return a.elt == KGE_ELT_F32 ? delta_scan_t<float>(a, st) : delta_scan_t<__nv_bfloat16>(a, st);
}

}  // namespace kge

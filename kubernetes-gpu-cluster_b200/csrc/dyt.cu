// Dynamic Tanh in the place of norms for layer-list models: y = tanh(alpha x) * w + b, element by element.  As it needs no
// statistics of the row, the pass that adds a sublayer's result to the fp32 residual stream (or that reads the embedding)
// writes the next sublayer's input along with it.  A result may come as rows, as two sides with a norm of their own each
// (the one case in which a row is read twice), or as routed experts' rows gathered by (token, choice) pair; a token's
// sources are summed in a fixed order whatever else is in the launch.
#include <algorithm>

#include "common.cuh"
#include "elt_access.cuh"
#include "hybrid_ops.h"

namespace kge {

namespace {

constexpr int DYT_MAX_THREADS = 256;

// one block per row; VEC: four neighbouring columns per thread and pass
template <typename E, bool VEC>
__global__ void __launch_bounds__(DYT_MAX_THREADS) dyt_f32in_kernel(E* y, const float* x, const int32_t* rows, float alpha, const E* w, const E* b, int d) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int W = VEC ? 4 : 1;
  const int r = blockIdx.x;
  const float* src = x + (int64_t)(rows ? rows[r] : r) * d;
  for (int c = threadIdx.x * W; c < d; c += blockDim.x * W) {
    float v[4], wv[4], bv[4];
    if (VEC) { ld4(src + c, v); ld4(w + c, wv); ld4(b + c, bv); } else { v[0] = src[c]; wv[0] = ldf(w + c); bv[0] = ldf(b + c); }
#pragma unroll
    for (int k = 0; k < W; ++k) v[k] = fmaf(tanhf(alpha * v[k]), wv[k], bv[k]);
    if (VEC) st4(y + (int64_t)r * d + c, v); else stf(y + (int64_t)r * d + c, v[0]);
  }
}

// INNER: sources with a norm of their own (their sums of squares first, then a second read of the rows)
template <typename E, bool VEC, bool INNER>
__global__ void __launch_bounds__(DYT_MAX_THREADS) dyt_combine_kernel(DytCombineArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int W = VEC ? 4 : 1;
  __shared__ float red[33];
  const int t = blockIdx.x, d = a.d;
  float f[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) f[i] = i < a.nsrc ? (a.rscale[i] ? a.src_scale * a.rscale[i][t] : a.src_scale) : 0.f;
  if (INNER) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      if (i >= a.nsrc || !a.inner_w[i]) continue;
      const E* s = (const E*)a.src[i] + (int64_t)t * a.ld[i];
      float ss = 0.f;
      for (int c = threadIdx.x * W; c < d; c += blockDim.x * W) {
        float v[4];
        if (VEC) ld4(s + c, v); else v[0] = ldf(s + c);
#pragma unroll
        for (int k = 0; k < W; ++k) ss = fmaf(v[k], v[k], ss);
      }
      f[i] *= 1.f / sqrtf(block_sum(ss, red) / (float)d + a.eps);
    }
  }
  float* res = a.res + (int64_t)t * d;
  const E* emb = a.table ? (const E*)a.table + (int64_t)a.ids[t] * d : nullptr;
  const int32_t* pr = a.pair_row ? a.pair_row + (int64_t)t * a.top : nullptr;
  const float* pw = a.pair_row ? a.pair_w + (int64_t)t * a.top : nullptr;
  for (int c = threadIdx.x * W; c < d; c += blockDim.x * W) {
    float r[4], s[4] = {0.f, 0.f, 0.f, 0.f};
    if (emb) {
      if (VEC) ld4(emb + c, r); else r[0] = ldf(emb + c);
#pragma unroll
      for (int k = 0; k < W; ++k) r[k] *= a.table_scale;
    } else if (VEC) ld4(res + c, r); else r[0] = res[c];
    if (pr) {
#pragma unroll 4
      for (int q = 0; q < a.top; ++q) {
        const E* src = (const E*)a.pair_src + (int64_t)pr[q] * d + c;
        const float wq = pw[q];
        float v[4];
        if (VEC) ld4(src, v); else v[0] = ldf(src);
#pragma unroll
        for (int k = 0; k < W; ++k) s[k] = fmaf(wq, v[k], s[k]);
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      if (i >= a.nsrc) continue;
      float v[4], wv[4] = {1.f, 1.f, 1.f, 1.f};
      const E* src = (const E*)a.src[i] + (int64_t)t * a.ld[i] + c;
      if (VEC) ld4(src, v); else v[0] = ldf(src);
      if (INNER && a.inner_w[i]) { if (VEC) ld4((const E*)a.inner_w[i] + c, wv); else wv[0] = ldf((const E*)a.inner_w[i] + c); }
#pragma unroll
      for (int k = 0; k < W; ++k) s[k] = fmaf(INNER ? v[k] * f[i] : f[i], INNER ? wv[k] : v[k], s[k]);
    }
#pragma unroll
    for (int k = 0; k < W; ++k) r[k] += s[k];
    if (VEC) st4(res + c, r); else res[c] = r[0];
    if (a.next_y) {
      E* ny = (E*)a.next_y + (int64_t)t * d + c;
      float wv[4], bv[4], o[4];
      if (VEC) { ld4((const E*)a.next_w + c, wv); ld4((const E*)a.next_b + c, bv); } else { wv[0] = ldf((const E*)a.next_w + c); bv[0] = ldf((const E*)a.next_b + c); }
#pragma unroll
      for (int k = 0; k < W; ++k) o[k] = fmaf(tanhf(a.next_alpha * r[k]), wv[k], bv[k]);
      if (VEC) st4(ny, o); else stf(ny, o[0]);
    }
  }
}

bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
int row_threads(int d, bool vec) { return std::max(32, std::min(DYT_MAX_THREADS, ((vec ? d / 4 : d) + 31) / 32 * 32)); }

template <typename E>
cudaError_t launch_combine(const DytCombineArgs& a, bool vec, bool inner, cudaStream_t st) {
  const dim3 grid(a.T), block(row_threads(a.d, vec));
  if (inner) return vec ? launch_pdl(dyt_combine_kernel<E, true, true>, grid, block, 0, st, a) : launch_pdl(dyt_combine_kernel<E, false, true>, grid, block, 0, st, a);
  return vec ? launch_pdl(dyt_combine_kernel<E, true, false>, grid, block, 0, st, a) : launch_pdl(dyt_combine_kernel<E, false, false>, grid, block, 0, st, a);
}

}  // namespace

int dyt_f32in(void* y, const float* x, const int32_t* rows, float alpha, const void* w, const void* b, int R, int d, int elt, cudaStream_t st) {
  if (R <= 0) return 0;
  KGE_REQUIRE(y && x && w && b && d > 0, "dyt_f32in: bad arguments");
  const bool vec = d % 4 == 0 && al16(y) && al16(x) && al16(w) && al16(b);
  const dim3 grid(R), block(row_threads(d, vec));
  cudaError_t ce;
  if (elt == KGE_ELT_F32)
    ce = vec ? launch_pdl(dyt_f32in_kernel<float, true>, grid, block, 0, st, (float*)y, x, rows, alpha, (const float*)w, (const float*)b, d)
             : launch_pdl(dyt_f32in_kernel<float, false>, grid, block, 0, st, (float*)y, x, rows, alpha, (const float*)w, (const float*)b, d);
  else
    ce = vec ? launch_pdl(dyt_f32in_kernel<__nv_bfloat16, true>, grid, block, 0, st, (__nv_bfloat16*)y, x, rows, alpha, (const __nv_bfloat16*)w, (const __nv_bfloat16*)b, d)
             : launch_pdl(dyt_f32in_kernel<__nv_bfloat16, false>, grid, block, 0, st, (__nv_bfloat16*)y, x, rows, alpha, (const __nv_bfloat16*)w, (const __nv_bfloat16*)b, d);
  KGE_CUDA_OK(ce);
  return 0;
}

int dyt_combine(const DytCombineArgs& a, cudaStream_t st) {
  if (a.T <= 0) return 0;
  KGE_REQUIRE(a.res && a.d > 0 && a.nsrc >= 0 && a.nsrc <= 2 && (!a.table || a.ids) && (!a.pair_row || (a.pair_src && a.pair_w && a.top > 0)) &&
              (!a.next_y || (a.next_w && a.next_b)), "dyt_combine: bad arguments");
  bool vec = a.d % 4 == 0 && al16(a.res) && al16(a.table) && al16(a.pair_src) && al16(a.next_w) && al16(a.next_b) && al16(a.next_y), inner = false;
  for (int i = 0; i < a.nsrc; ++i) {
    vec = vec && a.ld[i] % 4 == 0 && al16(a.src[i]) && al16(a.inner_w[i]);
    inner = inner || a.inner_w[i];
  }
  KGE_CUDA_OK(a.elt == KGE_ELT_F32 ? launch_combine<float>(a, vec, inner, st) : launch_combine<__nv_bfloat16>(a, vec, inner, st));
  return 0;
}

}  // namespace kge

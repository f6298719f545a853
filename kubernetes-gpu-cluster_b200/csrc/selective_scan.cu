// Selective scan for layer-list models: every channel c carries N fp32 numbers that decay and are written at a rate of the
// token's own,
//     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,      y_c = sum_n S[c, n] C_n + D_c x_c,      out_c = y_c silu(z_c).
// The state lives in the request's slot between steps, so a prompt cut anywhere continues exactly.
//   prompt steps: KQ neighbouring lanes share a channel and walk its request's rows in order with NPT states each in registers;
//     the rows' operands are staged CT tokens at a time, the next stage's being requested while one is computed.  Sums over n of
//     four tokens are exchanged together, so that every lane ends with one token's sum and finishes that token's output.
//   single tokens: a thread owns four neighbouring states of a channel for several requests; what it moves is the state.
#include <algorithm>
#include <type_traits>

#include "common.cuh"
#include "elt_access.cuh"
#include "f32x2.cuh"
#include "hybrid_ops.h"

namespace kge {

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float ex2(float v) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v)); return r; }
// exp(v) of an exponent that 16-bit engines hold in units of log 2.  A slowly decaying state is multiplied by numbers just below 1
// thousands of times, where an exponential that errs by a unit in the last place on one side adds up; float32 engines round
// the exact one to nearest.
template <typename E> __device__ __forceinline__ float decay_exp(float v) {
  if constexpr (std::is_same<E, float>::value) return (float)exp((double)v);
  else return ex2(v);
}
template <typename E> __device__ __forceinline__ float silu_f(float v) { return std::is_same<E, float>::value ? v / (1.f + expf(-v)) : __fdividef(v, 1.f + ex2(-LOG2E * v)); }

constexpr int SS_THREADS = 64;

template <typename E, int KQ, int NPT, int CT>
__global__ void __launch_bounds__(SS_THREADS) selective_scan_kernel(SelectiveScanArgs a) {
  pdl_launch_dependents();
  constexpr int CH = SS_THREADS / KQ, NW = KQ * NPT, NP = NPT / 2;
  constexpr int PBC = CT * NW / SS_THREADS, PCH = CT * CH / SS_THREADS > 0 ? CT * CH / SS_THREADS : 1;
  __shared__ __align__(16) float Bs[CT][NW], Cs[CT][NW], xs[CT][CH], ds[CT][CH], zs[CT][CH];
  const int tid = threadIdx.x, kq = tid % KQ, ch = tid / KQ, c0 = blockIdx.x * CH, c = c0 + ch, b = blockIdx.y, N = a.N, C = a.C;
  const bool on = c < C;
  // the coefficients do not depend on the kernel before this one
  f2 A2[NP];
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int n = kq * NPT + 2 * i;
    constexpr float s = std::is_same<E, float>::value ? 1.f : LOG2E;
    A2[i] = pk(on && n < N ? a.A[(int64_t)c * N + n] * s : 0.f, on && n + 1 < N ? a.A[(int64_t)c * N + n + 1] * s : 0.f);
  }
  const float D = on ? a.D[c] : 0.f;
  pdl_wait();
  const int r0 = a.qsl[b], r1 = a.qsl[b + 1];
  if (r0 >= r1) return;
  const bool fresh = a.positions[r0] == 0;
  float* Sg = a.state + (int64_t)a.slots[b] * a.slot_stride + (int64_t)c * N + kq * NPT;
  f2 S[NP];
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int n = kq * NPT + 2 * i;
    S[i] = pk(on && !fresh && n < N ? Sg[2 * i] : 0.f, on && !fresh && n + 1 < N ? Sg[2 * i + 1] : 0.f);
  }
  // the next stage's operands, in registers: this thread's share of the B and C rows and of the channels' x, dt and z
  float fb[PBC], fc[PBC], fx[PCH], fd[PCH], fz[PCH];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < PBC; ++i) {
      const int e = i * SS_THREADS + tid, t = t0 + e / NW, n = e % NW;
      const bool ok = t < r1 && n < N;
      fb[i] = ok ? ldf((const E*)a.b + (int64_t)t * a.ldbc + n) : 0.f;
      fc[i] = ok ? ldf((const E*)a.c + (int64_t)t * a.ldbc + n) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < PCH; ++i) {
      const int e = i * SS_THREADS + tid, t = t0 + e / CH, k = c0 + e % CH;
      const bool ok = e < CT * CH && t < r1 && k < C;
      fx[i] = ok ? ldf((const E*)a.x + (int64_t)t * a.ldx + k) : 0.f;
      fd[i] = ok ? a.dt[(int64_t)t * a.lddt + k] : 0.f;      // a row beyond the request leaves the state as it is
      fz[i] = ok ? ldf((const E*)a.z + (int64_t)t * a.ldz + k) : 0.f;
    }
  };
  fetch(r0);
  for (int t0 = r0; t0 < r1; t0 += CT) {
    __syncthreads();                                 // the previous stage's readers are done
#pragma unroll
    for (int i = 0; i < PBC; ++i) {
      const int e = i * SS_THREADS + tid;
      Bs[e / NW][e % NW] = fb[i]; Cs[e / NW][e % NW] = fc[i];
    }
#pragma unroll
    for (int i = 0; i < PCH; ++i) {
      const int e = i * SS_THREADS + tid;
      if (e < CT * CH) { xs[e / CH][e % CH] = fx[i]; ds[e / CH][e % CH] = fd[i]; zs[e / CH][e % CH] = fz[i]; }
    }
    __syncthreads();
    if (t0 + CT < r1) fetch(t0 + CT);
    const int n = min(CT, r1 - t0);
#pragma unroll 1
    for (int q = 0; q < n; q += 4) {
      float y[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float dt = ds[q + u][ch], dx = dt * xs[q + u][ch];
        const f2 dt2 = pk(dt, dt), dx2 = pk(dx, dx);
        const f2 *B2 = reinterpret_cast<const f2*>(&Bs[q + u][kq * NPT]), *C2 = reinterpret_cast<const f2*>(&Cs[q + u][kq * NPT]);
        f2 acc = 0ull;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
          float e0, e1;
          upk(mul2(dt2, A2[i]), e0, e1);
          S[i] = fma2(pk(decay_exp<E>(e0), decay_exp<E>(e1)), S[i], mul2(dx2, B2[i]));
          acc = fma2(S[i], C2[i], acc);
        }
        y[u] = sum2(acc);
      }
      // four tokens' sums over the KQ lanes: two exchanges leave each lane with token kq % 4, the rest add up
      const bool o0 = kq & 1, o1 = kq & 2;
      const float s0 = (o0 ? y[1] : y[0]) + __shfl_xor_sync(0xffffffffu, o0 ? y[0] : y[1], 1);
      const float s1 = (o0 ? y[3] : y[2]) + __shfl_xor_sync(0xffffffffu, o0 ? y[2] : y[3], 1);
      float s = (o1 ? s1 : s0) + __shfl_xor_sync(0xffffffffu, o1 ? s0 : s1, 2);
#pragma unroll
      for (int off = 4; off < KQ; off <<= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
      const int u = q + (kq & 3);
      if (on && kq < 4 && u < n) stf((E*)a.out + (int64_t)(t0 + u) * a.ldo + c, fmaf(D, xs[u][ch], s) * silu_f<E>(zs[u][ch]));
    }
  }
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int n = kq * NPT + 2 * i;
    float x, y;
    upk(S[i], x, y);
    if (on && n < N) Sg[2 * i] = x;
    if (on && n + 1 < N) Sg[2 * i + 1] = y;
  }
}

// The same walk for bfloat16 rows in whole 16-byte pieces (channels, states, strides and offsets multiples of 8): a thread requests the
// next stage's pieces as they are and converts B and C once, on their way to shared memory.
template <int KQ, int NPT, int CT>
__global__ void __launch_bounds__(SS_THREADS) selective_scan_vec_kernel(SelectiveScanArgs a) {
  pdl_launch_dependents();
  typedef __nv_bfloat16 E;
  constexpr int CH = SS_THREADS / KQ, NW = KQ * NPT, NP = NPT / 2;
  constexpr int NBC = 2 * CT * NW / 8, NX = CT * CH / 8, ND = CT * CH / 4;      // 16-byte pieces of a stage: B and C rows, x (and z) rows, dt rows
  constexpr int PB = NBC / SS_THREADS, PX = (2 * NX + SS_THREADS - 1) / SS_THREADS, PD = (ND + SS_THREADS - 1) / SS_THREADS;
  static_assert(NBC % SS_THREADS == 0 && CH % 8 == 0, "pieces");
  __shared__ __align__(16) float BCs[CT][2 * NW], ds[CT][CH];
  __shared__ __align__(16) E xz[2][CT][CH];
  const int tid = threadIdx.x, kq = tid % KQ, ch = tid / KQ, c0 = blockIdx.x * CH, c = c0 + ch, b = blockIdx.y, N = a.N, C = a.C;
  const bool on = c < C;
  f2 A2[NP];
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int n = kq * NPT + 2 * i;
    A2[i] = pk(on && n < N ? a.A[(int64_t)c * N + n] * LOG2E : 0.f, on && n + 1 < N ? a.A[(int64_t)c * N + n + 1] * LOG2E : 0.f);
  }
  const float D = on ? a.D[c] : 0.f;
  pdl_wait();
  const int r0 = a.qsl[b], r1 = a.qsl[b + 1];
  if (r0 >= r1) return;
  const bool fresh = a.positions[r0] == 0;
  float* Sg = a.state + (int64_t)a.slots[b] * a.slot_stride + (int64_t)c * N + kq * NPT;
  f2 S[NP];
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int n = kq * NPT + 2 * i;
    S[i] = pk(on && !fresh && n < N ? Sg[2 * i] : 0.f, on && !fresh && n + 1 < N ? Sg[2 * i + 1] : 0.f);
  }
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  uint4 pb[PB], px[PX], pd[PD];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < PB; ++i) {
      const int e = i * SS_THREADS + tid, t = t0 + e / (NW / 4), q = e % (NW / 4), n = q % (NW / 8) * 8;
      const E* src = (const E*)(q < NW / 8 ? a.b : a.c) + (int64_t)t * a.ldbc + n;
      pb[i] = t < r1 && n < N ? *reinterpret_cast<const uint4*>(src) : zero;
    }
#pragma unroll
    for (int i = 0; i < PX; ++i) {
      const int e = i * SS_THREADS + tid, z = e / NX, f = e % NX, t = t0 + f / (CH / 8), k = c0 + f % (CH / 8) * 8;
      px[i] = e < 2 * NX && t < r1 && k < C ? *reinterpret_cast<const uint4*>(z ? (const E*)a.z + (int64_t)t * a.ldz + k : (const E*)a.x + (int64_t)t * a.ldx + k) : zero;
    }
#pragma unroll
    for (int i = 0; i < PD; ++i) {
      const int e = i * SS_THREADS + tid, t = t0 + e / (CH / 4), k = c0 + e % (CH / 4) * 4;
      pd[i] = e < ND && t < r1 && k < C ? *reinterpret_cast<const uint4*>(a.dt + (int64_t)t * a.lddt + k) : zero;      // a row beyond the request leaves the state as it is
    }
  };
  fetch(r0);
  for (int t0 = r0; t0 < r1; t0 += CT) {
    __syncthreads();                                 // the previous stage's readers are done
#pragma unroll
    for (int i = 0; i < PB; ++i) {
      const int e = i * SS_THREADS + tid;
      float* dst = &BCs[e / (NW / 4)][e % (NW / 4) * 8];
      *reinterpret_cast<float4*>(dst) = make_float4(__uint_as_float(pb[i].x << 16), __uint_as_float(pb[i].x & 0xffff0000u), __uint_as_float(pb[i].y << 16), __uint_as_float(pb[i].y & 0xffff0000u));
      *reinterpret_cast<float4*>(dst + 4) = make_float4(__uint_as_float(pb[i].z << 16), __uint_as_float(pb[i].z & 0xffff0000u), __uint_as_float(pb[i].w << 16), __uint_as_float(pb[i].w & 0xffff0000u));
    }
#pragma unroll
    for (int i = 0; i < PX; ++i) {
      const int e = i * SS_THREADS + tid;
      if (e < 2 * NX) reinterpret_cast<uint4*>(&xz[0][0][0])[e] = px[i];
    }
#pragma unroll
    for (int i = 0; i < PD; ++i) {
      const int e = i * SS_THREADS + tid;
      if (e < ND) reinterpret_cast<uint4*>(&ds[0][0])[e] = pd[i];
    }
    __syncthreads();
    if (t0 + CT < r1) fetch(t0 + CT);
    const int n = min(CT, r1 - t0);
#pragma unroll 2
    for (int q = 0; q < n; q += 4) {
      float y[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float dt = ds[q + u][ch], dx = dt * __bfloat162float(xz[0][q + u][ch]);
        const f2 dt2 = pk(dt, dt), dx2 = pk(dx, dx);
        f2 acc = 0ull;
#pragma unroll
        for (int i = 0; i < NP; i += 2) {
          const ulonglong2 B2 = *reinterpret_cast<const ulonglong2*>(&BCs[q + u][kq * NPT + 2 * i]), C2 = *reinterpret_cast<const ulonglong2*>(&BCs[q + u][NW + kq * NPT + 2 * i]);
          float e0, e1, e2, e3;
          upk(mul2(dt2, A2[i]), e0, e1);
          upk(mul2(dt2, A2[i + 1]), e2, e3);
          S[i] = fma2(pk(ex2(e0), ex2(e1)), S[i], mul2(dx2, B2.x));
          S[i + 1] = fma2(pk(ex2(e2), ex2(e3)), S[i + 1], mul2(dx2, B2.y));
          acc = fma2(S[i], C2.x, acc);
          acc = fma2(S[i + 1], C2.y, acc);
        }
        y[u] = sum2(acc);
      }
      const bool o0 = kq & 1, o1 = kq & 2;           // sums over the KQ lanes as above
      const float s0 = (o0 ? y[1] : y[0]) + __shfl_xor_sync(0xffffffffu, o0 ? y[0] : y[1], 1);
      const float s1 = (o0 ? y[3] : y[2]) + __shfl_xor_sync(0xffffffffu, o0 ? y[2] : y[3], 1);
      float s = (o1 ? s1 : s0) + __shfl_xor_sync(0xffffffffu, o1 ? s0 : s1, 2);
#pragma unroll
      for (int off = 4; off < KQ; off <<= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
      const int u = q + (kq & 3);
      if (on && kq < 4 && u < n)
        ((E*)a.out)[(int64_t)(t0 + u) * a.ldo + c] = __float2bfloat16_rn(fmaf(D, __bfloat162float(xz[0][u][ch]), s) * silu_f<E>(__bfloat162float(xz[1][u][ch])));
    }
  }
#pragma unroll
  for (int i = 0; i < NP; ++i) {
    const int n = kq * NPT + 2 * i;
    float x, y;
    upk(S[i], x, y);
    if (on && n < N) Sg[2 * i] = x;
    if (on && n + 1 < N) Sg[2 * i + 1] = y;
  }
}

// one row per request (row b belongs to request b): NQ = N / 4 neighbouring lanes hold a channel, RPT requests per thread
template <typename E, int RPT>
__global__ void __launch_bounds__(256) selective_step_kernel(SelectiveScanArgs a, int NQ) {
  pdl_launch_dependents();
  const int64_t idx = (int64_t)blockIdx.x * 256 + threadIdx.x;
  const int c = (int)(idx / NQ), nq = (int)(idx % NQ), b0 = blockIdx.y * RPT;
  const bool on = c < a.C;
  constexpr float sc = std::is_same<E, float>::value ? 1.f : LOG2E;
  float A[4] = {0.f, 0.f, 0.f, 0.f}, D = 0.f;
  if (on) { ld4(a.A + (int64_t)c * a.N + nq * 4, A); D = a.D[c]; }
  pdl_wait();
  float S[RPT][4], B[RPT][4], Cv[RPT][4], x[RPT], dt[RPT], z[RPT];
  float* Sg[RPT];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int b = b0 + r;
    if (!on || b >= a.B) continue;
    Sg[r] = a.state + (int64_t)a.slots[b] * a.slot_stride + (int64_t)c * a.N + nq * 4;
    if (a.positions[b] == 0) S[r][0] = S[r][1] = S[r][2] = S[r][3] = 0.f; else ld4(Sg[r], S[r]);
    ld4((const E*)a.b + (int64_t)b * a.ldbc + nq * 4, B[r]); ld4((const E*)a.c + (int64_t)b * a.ldbc + nq * 4, Cv[r]);
    x[r] = ldf((const E*)a.x + (int64_t)b * a.ldx + c); z[r] = ldf((const E*)a.z + (int64_t)b * a.ldz + c); dt[r] = a.dt[(int64_t)b * a.lddt + c];
  }
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int b = b0 + r;
    float y = 0.f;
    if (on && b < a.B) {
      const float dx = dt[r] * x[r];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        S[r][k] = fmaf(decay_exp<E>(dt[r] * (A[k] * sc)), S[r][k], dx * B[r][k]);
        y = fmaf(S[r][k], Cv[r][k], y);
      }
      st4(Sg[r], S[r]);
    }
    for (int off = 1; off < NQ; off <<= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
    if (on && b < a.B && nq == 0) stf((E*)a.out + (int64_t)b * a.ldo + c, fmaf(D, x[r], y) * silu_f<E>(z[r]));
  }
}

template <typename E, int KQ, int NPT, int CT>
cudaError_t launch_scan(const SelectiveScanArgs& a, cudaStream_t st) {
  constexpr int CH = SS_THREADS / KQ;
  return launch_pdl(selective_scan_kernel<E, KQ, NPT, CT>, dim3((a.C + CH - 1) / CH, a.B), dim3(SS_THREADS), 0, st, a);
}

template <int KQ, int NPT, int CT>
cudaError_t launch_scan_vec(const SelectiveScanArgs& a, cudaStream_t st) {
  constexpr int CH = SS_THREADS / KQ;
  return launch_pdl(selective_scan_vec_kernel<KQ, NPT, CT>, dim3((a.C + CH - 1) / CH, a.B), dim3(SS_THREADS), 0, st, a);
}

template <typename E>
cudaError_t dispatch(const SelectiveScanArgs& a, cudaStream_t st) {
  const int NQ = a.N / 4;
  if (a.T == a.B && a.N % 4 == 0 && NQ <= 32 && (NQ & (NQ - 1)) == 0 && a.ldbc % 4 == 0 && a.slot_stride % 4 == 0 &&
      ((reinterpret_cast<uintptr_t>(a.state) | reinterpret_cast<uintptr_t>(a.A)) & 15) == 0 &&
      ((reinterpret_cast<uintptr_t>(a.b) | reinterpret_cast<uintptr_t>(a.c)) & (4 * sizeof(E) - 1)) == 0) {
    const unsigned gx = (unsigned)(((int64_t)a.C * NQ + 255) / 256);
    return a.B >= 16 ? launch_pdl(selective_step_kernel<E, 4>, dim3(gx, (a.B + 3) / 4), dim3(256), 0, st, a, NQ)
                     : launch_pdl(selective_step_kernel<E, 1>, dim3(gx, a.B), dim3(256), 0, st, a, NQ);
  }
  auto al16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  if (std::is_same<E, __nv_bfloat16>::value && a.N % 8 == 0 && a.N <= 64 && a.C % 8 == 0 && a.ldx % 8 == 0 && a.ldz % 8 == 0 && a.ldbc % 8 == 0 && a.lddt % 4 == 0 && al16(a.x) && al16(a.z) &&
      al16(a.b) && al16(a.c) && al16(a.dt))
    return a.N <= 16 ? launch_scan_vec<4, 4, 32>(a, st) : a.N <= 32 ? launch_scan_vec<4, 8, 16>(a, st) : launch_scan_vec<8, 8, 16>(a, st);
  if (a.N <= 16) return launch_scan<E, 4, 4, 16>(a, st);
  if (a.N <= 32) return launch_scan<E, 4, 8, 16>(a, st);
  if (a.N <= 64) return launch_scan<E, 8, 8, 8>(a, st);
  if (a.N <= 128) return launch_scan<E, 16, 8, 8>(a, st);
  return launch_scan<E, 32, 8, 4>(a, st);
}

}  // namespace

int selective_scan(const SelectiveScanArgs& a, cudaStream_t st) {
  if (a.T <= 0) return 0;
  KGE_REQUIRE(a.C > 0 && a.N > 0 && a.N <= 256 && a.B <= 65535, "selective_scan: %d channels of %d numbers", a.C, a.N);
  KGE_CUDA_OK(a.elt == KGE_ELT_F32 ? dispatch<float>(a, st) : dispatch<__nv_bfloat16>(a, st));
  return 0;
}

}  // namespace kge

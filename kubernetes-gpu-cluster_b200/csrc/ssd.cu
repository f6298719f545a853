// State-space dual recurrence for layer-list models: each head carries an N x P matrix S in fp32 with one decay per token,
//     S <- a_t S + dt_t B_t x_t^T,      y_t = S^T C_t + D x_t,      dt_t = softplus(dt_pre + dt_bias),  a_t = exp(-exp(A_log) dt_t),
// B and C shared by the heads of a group.  S lives in the request's state slot between steps, so a prompt cut anywhere
// continues exactly.  Three kernels:
//   ssd_chunk_kernel (bfloat16, prompt steps): 64 tokens at a time.  With c_t the running sum of the chunk's log decays and S the
//     state at its start,
//         y_t = e^{c_t} S^T C_t + sum_{j <= t} e^{c_t - c_j} dt_j (C_t . B_j) x_j,      S <- e^{c_last} S + sum_j e^{c_last - c_j} dt_j B_j x_j^T.
//     Every exponent is <= 0; differences are formed from sums held as a pair of fp32 numbers.  The products run on the tensor
//     cores with fp32 accumulation: x, B and C are bfloat16 as they come; what is fp32 (the state, the weighted scores, the weighted
//     B) enters as three bfloat16 terms that together hold its 24 bits.  The state stays in fp32 registers across chunks.
//   ssd_step_kernel (one row per request): streams the state through registers once.
//   ssd_seq_kernel (any size, float32 storage): token by token, eight lanes per column.
#include <algorithm>
#include <type_traits>

#include "common.cuh"
#include "elt_access.cuh"
#include "hybrid_ops.h"

namespace kge {

namespace {

__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
// the decay of one token; float32 engines round the exact exponential to nearest (a slow decay is applied thousands of times)
template <typename E> __device__ __forceinline__ float decay_exp(float v) {
  if constexpr (std::is_same<E, float>::value) return (float)exp((double)v);
  else return expf(v);
}
__device__ __forceinline__ float fast_ex2(float v) { float r; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v)); return r; }

// ------------------------------------------------------------------------------------------------ one row per request
// Threads own (row group, four columns) pieces of the head's matrix; IPT pieces are requested together.
template <typename E>
__global__ void __launch_bounds__(256) ssd_step_kernel(SsdArgs a) {
  pdl_launch_dependents();
  constexpr int IPT = 8;
  __shared__ __align__(16) float red[256][4];
  const int h = blockIdx.x, b = blockIdx.y, g = h / (a.H / a.G), PQ = a.P / 4, RG = 256 / PQ, tid = threadIdx.x, rg = tid / PQ, pq = tid % PQ;
  const float coef = a.a_coef[h], bias = a.dt_bias[h], D = a.D[h];
  pdl_wait();
  const bool fresh = a.positions[b] == 0, on = rg < RG;
  float* Sg = a.state + (int64_t)a.slots[b] * a.slot_stride + (int64_t)h * a.N * a.P + pq * 4;
  const E *Bp = (const E*)a.b + (int64_t)b * a.ld + g * a.N, *Cp = (const E*)a.c + (int64_t)b * a.ld + g * a.N;
  float y[4] = {0.f, 0.f, 0.f, 0.f}, x[4] = {0.f, 0.f, 0.f, 0.f}, dx[4];
  const float pre = ldf((const E*)a.dt_pre + (int64_t)b * a.lddt + h);
  if (on) {
#pragma unroll
    for (int k = 0; k < 4; ++k) x[k] = ldf((const E*)a.x + (int64_t)b * a.ld + h * a.P + pq * 4 + k);
  }
  for (int n0 = rg; n0 < a.N; n0 += RG * IPT) {
    float S[IPT][4], bv[IPT], cv[IPT];
#pragma unroll
    for (int i = 0; i < IPT; ++i) {
      const int n = n0 + i * RG;
      S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
      if (on && n < a.N) {
        if (!fresh) ld4(Sg + (int64_t)n * a.P, S[i]);
        bv[i] = ldf(Bp + n); cv[i] = ldf(Cp + n);
      }
    }
    const float dt = softplus_f(pre + bias), dec = decay_exp<E>(-coef * dt);
#pragma unroll
    for (int k = 0; k < 4; ++k) dx[k] = dt * x[k];
#pragma unroll
    for (int i = 0; i < IPT; ++i) {
      const int n = n0 + i * RG;
      if (on && n < a.N) {
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          S[i][k] = fmaf(dec, S[i][k], bv[i] * dx[k]);
          y[k] = fmaf(S[i][k], cv[i], y[k]);
        }
        st4(Sg + (int64_t)n * a.P, S[i]);
      }
    }
  }
  st4(red[tid], y);
  __syncthreads();
  for (int p = tid; p < a.P; p += 256) {
    float s = 0.f;
    for (int r = 0; r < RG; ++r) s += red[r * PQ + p / 4][p & 3];
    a.o32[((int64_t)b * a.H + h) * a.P + p] = fmaf(D, ldf((const E*)a.x + (int64_t)b * a.ld + h * a.P + p), s);
  }
}

// ------------------------------------------------------------------------------------------------ any size
constexpr int SQ_CT = 16, SQ_COLS = 32;

template <typename E, int KPT>
__global__ void __launch_bounds__(256) ssd_seq_kernel(SsdArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float Bs[SQ_CT][8 * KPT], Cs[SQ_CT][8 * KPT], xs[SQ_CT][SQ_COLS], dts[SQ_CT], dec[SQ_CT];
  const int tid = threadIdx.x, kq = tid & 7, col = tid >> 3, h = blockIdx.y, b = blockIdx.z, g = h / (a.H / a.G), p = blockIdx.x * SQ_COLS + col;
  const int r0 = a.qsl[b], r1 = a.qsl[b + 1];
  if (r0 >= r1) return;
  const bool fresh = a.positions[r0] == 0, on = p < a.P;
  const float coef = a.a_coef[h], bias = a.dt_bias[h], D = a.D[h];
  float* Sg = a.state + (int64_t)a.slots[b] * a.slot_stride + (int64_t)h * a.N * a.P + p;
  float S[KPT];                                      // states n = i * 8 + kq
#pragma unroll
  for (int i = 0; i < KPT; ++i) { const int n = i * 8 + kq; S[i] = on && !fresh && n < a.N ? Sg[(int64_t)n * a.P] : 0.f; }
  for (int t0 = r0; t0 < r1; t0 += SQ_CT) {
    const int nt = min(SQ_CT, r1 - t0);
    __syncthreads();
    for (int e = tid; e < SQ_CT * 8 * KPT; e += 256) {
      const int t = e / (8 * KPT), n = e % (8 * KPT);
      const bool ok = t < nt && n < a.N;
      Bs[t][n] = ok ? ldf((const E*)a.b + (int64_t)(t0 + t) * a.ld + g * a.N + n) : 0.f;
      Cs[t][n] = ok ? ldf((const E*)a.c + (int64_t)(t0 + t) * a.ld + g * a.N + n) : 0.f;
    }
    for (int e = tid; e < SQ_CT * SQ_COLS; e += 256) {
      const int t = e / SQ_COLS, c = blockIdx.x * SQ_COLS + e % SQ_COLS;
      xs[t][e % SQ_COLS] = t < nt && c < a.P ? ldf((const E*)a.x + (int64_t)(t0 + t) * a.ld + h * a.P + c) : 0.f;
    }
    if (tid < nt) {
      const float dt = softplus_f(ldf((const E*)a.dt_pre + (int64_t)(t0 + tid) * a.lddt + h) + bias);
      dts[tid] = dt; dec[tid] = decay_exp<E>(-coef * dt);
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float x = xs[t][col], dx = dts[t] * x, d = dec[t];
      float y = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        S[i] = fmaf(d, S[i], dx * Bs[t][i * 8 + kq]);
        y = fmaf(S[i], Cs[t][i * 8 + kq], y);
      }
#pragma unroll
      for (int off = 1; off < 8; off <<= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
      if (on && kq == 0) a.o32[((int64_t)(t0 + t) * a.H + h) * a.P + p] = fmaf(D, x, y);
    }
  }
#pragma unroll
  for (int i = 0; i < KPT; ++i) { const int n = i * 8 + kq; if (on && n < a.N) Sg[(int64_t)n * a.P] = S[i]; }
}

// ------------------------------------------------------------------------------------------------ chunks of 64 tokens
constexpr int CL = 64, CP = 64, XPITCH = CP + 8;     // tokens per chunk, columns per block, row pitch of x and of the split state

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16 bytes from global to shared memory, or zeros
__device__ __forceinline__ void cp16z(void* dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0));
}
// two fp32 numbers as three pairs of bfloat16 that add up to their 24 bits
__device__ __forceinline__ void split3(float u, float v, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(u, v);
  const float2 hf = __bfloat1622float2(h);
  u -= hf.x; v -= hf.y;
  const __nv_bfloat162 m = __floats2bfloat162_rn(u, v);
  const float2 mf = __bfloat1622float2(m);
  const __nv_bfloat162 l = __floats2bfloat162_rn(u - mf.x, v - mf.y);
  hi = *reinterpret_cast<const uint32_t*>(&h); mid = *reinterpret_cast<const uint32_t*>(&m); lo = *reinterpret_cast<const uint32_t*>(&l);
}

template <int NPAD> struct ChunkSmem {
  static constexpr int BP = NPAD + 8;
  __nv_bfloat16 B[CL][BP], C[CL][BP], X[CL][XPITCH], S[3][NPAD][XPITCH];
  float hi[2][CL], lo[2][CL], dt[2][CL], w[2][CL], er[2][CL], etot[2];      // running sums (as pairs), steps, weights of the state's update, e^{c_t}
};

template <int NPAD>
__global__ void __launch_bounds__(256, 2) ssd_chunk_kernel(SsdArgs a, int ptiles) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t ssd_smem[];
  ChunkSmem<NPAD>& sm = *reinterpret_cast<ChunkSmem<NPAD>*>(ssd_smem);
  typedef __nv_bfloat16 E;
  constexpr int RT = NPAD / 16, SPLIT = 8 / RT, NT = 8 / SPLIT;      // the state: RT row tiles x SPLIT column parts over the eight warps, NT 8-column tiles each
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, cq = (lane & 3) * 2;
  const int h = blockIdx.x / ptiles, p0 = (blockIdx.x % ptiles) * CP, b = blockIdx.y, g = h / (a.H / a.G), N = a.N, P = min(CP, a.P - p0);
  const float coef = a.a_coef[h], bias = a.dt_bias[h], D = a.D[h];
  pdl_wait();
  const int r0 = a.qsl[b], r1 = a.qsl[b + 1];
  if (r0 >= r1) return;
  const bool fresh = a.positions[r0] == 0;
  float* Sg = a.state + (int64_t)a.slots[b] * a.slot_stride + (int64_t)h * N * a.P + p0;
  const E *xg = (const E*)a.x + h * a.P + p0, *bg = (const E*)a.b + g * N, *cg = (const E*)a.c + g * N;
  const int n0 = (warp % RT) * 16, sc0 = (warp / RT) * (NT * 8);     // this warp's tile of the state
  float S[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int n = n0 + gq + e * 8, p = sc0 + j * 8 + cq;
      float2 v = make_float2(0.f, 0.f);
      if (!fresh && n < N && p < P) v = *reinterpret_cast<const float2*>(Sg + (int64_t)n * a.P + p);
      S[j][e * 2] = v.x; S[j][e * 2 + 1] = v.y;
    }
  auto put_state = [&]() {                            // the state as three bfloat16 terms for the next chunk's read-out
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint32_t t3[3];
        split3(S[j][e * 2], S[j][e * 2 + 1], t3[0], t3[1], t3[2]);
#pragma unroll
        for (int k = 0; k < 3; ++k) *reinterpret_cast<uint32_t*>(&sm.S[k][n0 + gq + e * 8][sc0 + j * 8 + cq]) = t3[k];
      }
  };
  auto load_rows = [&](E* dst, int pitch, const E* src, int t0, int pieces, int valid) {
    for (int i = tid; i < CL * pieces; i += 256) {
      const int t = i / pieces, c = i % pieces;
      const bool ok = t0 + t < r1 && c < valid;
      cp16z(dst + t * pitch + c * 8, ok ? src + (int64_t)(t0 + t) * a.ld + c * 8 : src, ok);
    }
  };
  constexpr int BP = ChunkSmem<NPAD>::BP, NPC = NPAD / 8;
  load_rows(&sm.C[0][0], BP, cg, r0, NPC, N / 8);
  load_rows(&sm.B[0][0], BP, bg, r0, NPC, N / 8);
  load_rows(&sm.X[0][0], XPITCH, xg, r0, CP / 8, P / 8);
  asm volatile("cp.async.commit_group;");
  put_state();
  auto dt_raw = [&](int t) { return t < r1 ? ldf((const E*)a.dt_pre + (int64_t)t * a.lddt + h) : 0.f; };
  float raw0 = 0.f, raw1 = 0.f;                       // warp 0: the logits of two tokens per lane, a chunk ahead
  if (warp == 0) { raw0 = dt_raw(r0 + lane * 2); raw1 = dt_raw(r0 + lane * 2 + 1); }
  // read-out: 16 rows x 32 columns per warp; a row tile has more keys the later it lies, so the two halves run through them in opposite order
  const int rt = warp < 4 ? warp : 7 - warp, ct = (warp >> 2) * 32;
  const int lr = lane & 7, lm = lane >> 3;            // ldmatrix: row within a matrix, matrix
  // running sums, steps and weights of the chunk that starts at t0, into half s of their buffers (warp 0, two tokens per lane); the
  // logits of the chunk after it are requested
  auto scalars = [&](int t0, int s) {
    const int t = t0 + lane * 2;
    const float d0 = t < r1 ? softplus_f(raw0 + bias) : 0.f, d1 = t + 1 < r1 ? softplus_f(raw1 + bias) : 0.f;      // rows beyond the request: no step, no decay
    raw0 = dt_raw(t + CL); raw1 = dt_raw(t + CL + 1);
    const double l0 = (double)(-coef * d0) * 1.4426950408889634, l1 = (double)(-coef * d1) * 1.4426950408889634;
    double run = l0 + l1;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) { const double o = __shfl_up_sync(0xffffffffu, run, off); if (lane >= off) run += o; }
    const double c1 = run, c0 = run - l1, tot = __shfl_sync(0xffffffffu, run, 31);
    const float h0 = (float)c0, h1 = (float)c1;
    sm.hi[s][lane * 2] = h0; sm.hi[s][lane * 2 + 1] = h1;
    sm.lo[s][lane * 2] = (float)(c0 - (double)h0); sm.lo[s][lane * 2 + 1] = (float)(c1 - (double)h1);
    sm.dt[s][lane * 2] = d0; sm.dt[s][lane * 2 + 1] = d1;
    sm.w[s][lane * 2] = exp2f((float)(tot - c0)) * d0; sm.w[s][lane * 2 + 1] = exp2f((float)(tot - c1)) * d1;
    sm.er[s][lane * 2] = exp2f(h0); sm.er[s][lane * 2 + 1] = exp2f(h1);
    if (lane == 0) sm.etot[s] = exp2f((float)tot);
  };
  if (warp == 0) scalars(r0, 0);
  int s = 0;
  for (int t0 = r0; t0 < r1; t0 += CL, s ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int n = min(CL, r1 - t0);
    if (rt * 16 < n) {
      float y[4][4] = {};
      const E* crow = &sm.C[rt * 16 + (lm & 1) * 8 + lr][(lm >> 1) * 8];
      if (!(fresh && t0 == r0)) {                     // the carried state
#pragma unroll 2
        for (int ks = 0; ks < NPAD / 16; ++ks) {
          if (ks * 16 >= N) break;
          uint32_t af[4];
          ldsm4(af, crow + ks * 16);
#pragma unroll
          for (int k = 2; k >= 0; --k)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
              uint32_t bf[4];
              ldsm4t(bf, &sm.S[k][ks * 16 + (lm & 1) * 8 + lr][ct + j * 16 + (lm >> 1) * 8]);
              mma16816(y[j * 2], af, bf[0], bf[1]);
              mma16816(y[j * 2 + 1], af, bf[2], bf[3]);
            }
        }
        const float e0 = sm.er[s][rt * 16 + gq], e1 = sm.er[s][rt * 16 + gq + 8];
#pragma unroll
        for (int j = 0; j < 4; ++j) { y[j][0] *= e0; y[j][1] *= e0; y[j][2] *= e1; y[j][3] *= e1; }
      }
      const int ta = rt * 16 + gq, tb = ta + 8;
      const float ha = sm.hi[s][ta], la = sm.lo[s][ta], hb = sm.hi[s][tb], lb = sm.lo[s][tb];
      for (int kt = 0; kt <= rt; ++kt) {              // the chunk's own keys, 16 at a time
        float gs[2][4] = {};
#pragma unroll 4
        for (int ks = 0; ks < NPAD / 16; ++ks) {
          if (ks * 16 >= N) break;
          uint32_t af[4], bf[4];
          ldsm4(af, crow + ks * 16);
          ldsm4(bf, &sm.B[kt * 16 + (lm >> 1) * 8 + lr][ks * 16 + (lm & 1) * 8]);
          mma16816(gs[0], af, bf[0], bf[1]);
          mma16816(gs[1], af, bf[2], bf[3]);
        }
        uint32_t mf[3][4];
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int j0 = kt * 16 + q * 8 + cq, j1 = j0 + 1;
          const float h0 = sm.hi[s][j0], h1 = sm.hi[s][j1], l0 = sm.lo[s][j0], l1 = sm.lo[s][j1], d0 = sm.dt[s][j0], d1 = sm.dt[s][j1];
          const float v0 = j0 <= ta ? gs[q][0] * (fast_ex2((ha - h0) + (la - l0)) * d0) : 0.f, v1 = j1 <= ta ? gs[q][1] * (fast_ex2((ha - h1) + (la - l1)) * d1) : 0.f;
          const float v2 = j0 <= tb ? gs[q][2] * (fast_ex2((hb - h0) + (lb - l0)) * d0) : 0.f, v3 = j1 <= tb ? gs[q][3] * (fast_ex2((hb - h1) + (lb - l1)) * d1) : 0.f;
          split3(v0, v1, mf[0][q * 2], mf[1][q * 2], mf[2][q * 2]);
          split3(v2, v3, mf[0][q * 2 + 1], mf[1][q * 2 + 1], mf[2][q * 2 + 1]);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          uint32_t xf[4];
          ldsm4t(xf, &sm.X[kt * 16 + (lm & 1) * 8 + lr][ct + j * 16 + (lm >> 1) * 8]);
#pragma unroll
          for (int k = 2; k >= 0; --k) { mma16816(y[j * 2], mf[k], xf[0], xf[1]); mma16816(y[j * 2 + 1], mf[k], xf[2], xf[3]); }
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = ta + e * 8, p = ct + j * 8 + cq;
          if (t < n && p < P) {
            const float2 xv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&sm.X[t][p]));
            *reinterpret_cast<float2*>(a.o32 + ((int64_t)(t0 + t) * a.H + h) * a.P + p0 + p) = make_float2(fmaf(D, xv.x, y[j][e * 2]), fmaf(D, xv.y, y[j][e * 2 + 1]));
          }
        }
    }
    const bool more = t0 + CL < r1;
    if (warp == 0 && more) scalars(t0 + CL, s ^ 1);   // the warp with the shortest read-out
    __syncthreads();                                  // C and the split state have been read
    if (more) load_rows(&sm.C[0][0], BP, cg, t0 + CL, NPC, N / 8);
    {
      const float et = sm.etot[s];
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[j][e] *= et;
      if (n0 < N) {
        for (int ks = 0; ks < CL / 16; ++ks) {
          if (ks * 16 >= n) break;
          uint32_t bt[4], wf[3][4];
          ldsm4t(bt, &sm.B[ks * 16 + (lm >> 1) * 8 + lr][n0 + (lm & 1) * 8]);
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const int j0 = ks * 16 + (q >> 1) * 8 + cq;
            const float2 bv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&bt[q]));
            split3(bv.x * sm.w[s][j0], bv.y * sm.w[s][j0 + 1], wf[0][q], wf[1][q], wf[2][q]);
          }
#pragma unroll
          for (int j = 0; j < NT / 2; ++j) {
            uint32_t xf[4];
            ldsm4t(xf, &sm.X[ks * 16 + (lm & 1) * 8 + lr][sc0 + j * 16 + (lm >> 1) * 8]);
#pragma unroll
            for (int k = 2; k >= 0; --k) { mma16816(S[j * 2], wf[k], xf[0], xf[1]); mma16816(S[j * 2 + 1], wf[k], xf[2], xf[3]); }
          }
        }
      }
    }
    if (more) {
      put_state();
      __syncthreads();                                // B and x have been read
      load_rows(&sm.B[0][0], BP, bg, t0 + CL, NPC, N / 8);
      load_rows(&sm.X[0][0], XPITCH, xg, t0 + CL, CP / 8, P / 8);
      asm volatile("cp.async.commit_group;");
    }
  }
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int n = n0 + gq + e * 8, p = sc0 + j * 8 + cq;
      if (n < N && p < P) *reinterpret_cast<float2*>(Sg + (int64_t)n * a.P + p) = make_float2(S[j][e * 2], S[j][e * 2 + 1]);
    }
}

template <int NPAD>
int launch_chunk(const SsdArgs& a, cudaStream_t st) {
  const int ptiles = (a.P + CP - 1) / CP;
  constexpr size_t smem = sizeof(ChunkSmem<NPAD>);
  KGE_CUDA_OK(cudaFuncSetAttribute(ssd_chunk_kernel<NPAD>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  KGE_CUDA_OK(launch_pdl(ssd_chunk_kernel<NPAD>, dim3(a.H * ptiles, a.B), dim3(256), smem, st, a, ptiles));
  return 0;
}

template <typename E>
int dispatch(const SsdArgs& a, cudaStream_t st) {
  auto al = [](const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
  if (a.T == a.B && a.P % 4 == 0 && a.P <= 1024 && a.slot_stride % 4 == 0 && al(a.state, 16)) {
    KGE_CUDA_OK(launch_pdl(ssd_step_kernel<E>, dim3(a.H, a.B), dim3(256), 0, st, a));
    return 0;
  }
  if (std::is_same<E, __nv_bfloat16>::value && a.N <= 128 && a.N % 8 == 0 && a.P % 8 == 0 && a.ld % 8 == 0 && a.slot_stride % 2 == 0 && al(a.x, 16) && al(a.b, 16) && al(a.c, 16) &&
      al(a.state, 8) && al(a.o32, 8))
    return a.N <= 64 ? launch_chunk<64>(a, st) : launch_chunk<128>(a, st);
  const dim3 grid((a.P + SQ_COLS - 1) / SQ_COLS, a.H, a.B);
  KGE_CUDA_OK(a.N <= 32 ? launch_pdl(ssd_seq_kernel<E, 4>, grid, dim3(256), 0, st, a) : a.N <= 64 ? launch_pdl(ssd_seq_kernel<E, 8>, grid, dim3(256), 0, st, a)
              : a.N <= 128 ? launch_pdl(ssd_seq_kernel<E, 16>, grid, dim3(256), 0, st, a) : launch_pdl(ssd_seq_kernel<E, 32>, grid, dim3(256), 0, st, a));
  return 0;
}

}  // namespace

int ssd_scan(const SsdArgs& a, cudaStream_t st) {
  if (a.T <= 0) return 0;
  KGE_REQUIRE(a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.N > 0 && a.N <= 256 && a.P > 0 && a.H <= 65535 && a.B <= 65535, "ssd_scan: %d heads on %d groups of %d x %d", a.H, a.G, a.N, a.P);
  return a.elt == KGE_ELT_F32 ? dispatch<float>(a, st) : dispatch<__nv_bfloat16>(a, st);
}

}  // namespace kge

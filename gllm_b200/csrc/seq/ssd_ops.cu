// Kernels of the Mamba-2 mixer and of the parallel blocks around it (models/hybrid.py, block "parallel"): the
// state-space recurrence S <- exp(neg_a dt) S + dt b x^T, y = S^T c + d x with slot-indexed fp32 state as a one-token
// step and in chunked form on the tensor cores, the gate before a grouped RMS norm, the gated per-layer token input
// and cos / sin rows shared by the layers of a step.
//
// dt = softplus(dt + bias), the decays, their running sums and exponentials, the state and the norm are fp32 (sums of
// logarithms in two floats). Compiled WITHOUT --use_fast_math (build.py). Results of a row never depend on which
// other rows share the launch: every reduction has a fixed order.
#include <cuda_bf16.h>

#include "common/host_utils.h"
#include "seq/seq_common.cuh"

namespace {
using namespace seqk;
typedef __nv_bfloat16 bf16_t;

__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

// out[t, i] = cos(pos_t f_i), out[t, n + i] = sin(pos_t f_i); the angle in fp64
__global__ void rotary_angles_kernel(const int* __restrict__ positions, const double* __restrict__ freqs, int n,
                                     float* __restrict__ out, size_t total) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const size_t t = i / n, k = i - t * n;
  double sn, cs;
  sincos((double)positions[t] * freqs[k], &sn, &cs);
  out[t * 2 * n + k] = (float)cs;
  out[t * 2 * n + n + k] = (float)sn;
}

// out[t, i] = gelu_tanh(g[t, i]) * table[ids[t], col0 + i]
template <typename T>
__global__ void gelu_gate_embed_kernel(const T* __restrict__ g, long ldg, const int* __restrict__ ids, int vocab,
                                       const T* __restrict__ table, long ldt, int col0, T* __restrict__ out, int dim,
                                       size_t total) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  const size_t t = i / dim, c = i - t * dim;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const float z = to_f(g[t * ldg + c]);
  const float a = 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
  out[i] = from_f<T>(a * to_f(table[(size_t)id * ldt + col0 + c]));
}

// v = o * silu(gate); out = v / sqrt(mean over the group of v^2 + eps) * w. One block per (token, group); v is kept in
// shared memory between the two passes.
template <typename T>
__global__ void gate_then_norm_kernel(const float* __restrict__ o, int n, const T* __restrict__ gate, long ldg,
                                      const float* __restrict__ w, int group, float eps, T* __restrict__ out,
                                      long ldo) {
  extern __shared__ float sv[];
  __shared__ float red[32];
  const int t = blockIdx.x, c0 = blockIdx.y * group, nw = blockDim.x >> 5;
  const float* src = o + (size_t)t * n + c0;
  const T* gr = gate + (size_t)t * ldg + c0;
  float ss = 0.f;
  for (int i = threadIdx.x; i < group; i += blockDim.x) {
    const float z = to_f(gr[i]);
    const float v = src[i] * (z / (1.0f + expf(-z)));
    sv[i] = v;
    ss += v * v;
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < nw; ++i) tot += red[i];
  const float r = 1.0f / sqrtf(tot / (float)group + eps);
  T* dst = out + (size_t)t * ldo + c0;
  for (int i = threadIdx.x; i < group; i += blockDim.x) dst[i] = from_f<T>(sv[i] * r * w[c0 + i]);
}

// bf16 rows with everything 16-byte aligned: a thread keeps up to MAXV 4-wide pieces of the group in registers
template <int MAXV>
__global__ void __launch_bounds__(256) gate_then_norm_vec_kernel(
    const float* __restrict__ o, int n, const bf16_t* __restrict__ gate, long ldg, const float* __restrict__ w,
    int group, float eps, bf16_t* __restrict__ out, long ldo) {
  __shared__ float red[8];
  const int t = blockIdx.x, c0 = blockIdx.y * group, nw = blockDim.x >> 5, step = blockDim.x * 4;
  const float* src = o + (size_t)t * n + c0;
  const bf16_t* gr = gate + (size_t)t * ldg + c0;
  float4 v[MAXV];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < MAXV; ++k) {
    const int i = threadIdx.x * 4 + k * step;
    if (i < group) {
      float4 x = *reinterpret_cast<const float4*>(src + i);
      const uint2 gb = *reinterpret_cast<const uint2*>(gr + i);
      const float2 g0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gb.x));
      const float2 g1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gb.y));
      x.x *= g0.x / (1.0f + expf(-g0.x));
      x.y *= g0.y / (1.0f + expf(-g0.y));
      x.z *= g1.x / (1.0f + expf(-g1.x));
      x.w *= g1.y / (1.0f + expf(-g1.y));
      v[k] = x;
      ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    }
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int i = 0; i < nw; ++i) tot += red[i];
  const float r = 1.0f / sqrtf(tot / (float)group + eps);
  bf16_t* dst = out + (size_t)t * ldo + c0;
#pragma unroll
  for (int k = 0; k < MAXV; ++k) {
    const int i = threadIdx.x * 4 + k * step;
    if (i < group) {
      const float4 ww = *reinterpret_cast<const float4*>(w + c0 + i);
      const __nv_bfloat162 a = __floats2bfloat162_rn(v[k].x * r * ww.x, v[k].y * r * ww.y);
      const __nv_bfloat162 b = __floats2bfloat162_rn(v[k].z * r * ww.z, v[k].w * r * ww.w);
      uint2 ov;
      ov.x = *reinterpret_cast<const uint32_t*>(&a);
      ov.y = *reinterpret_cast<const uint32_t*>(&b);
      *reinterpret_cast<uint2*>(dst + i) = ov;
    }
  }
}

// One token per sequence: the state matrix [N, V] of a (sequence, head) is read, updated and written once with 16-byte
// accesses. A thread owns 4 value columns and every (256 / (V / 4))-th state row, ROWS rows in flight; partial
// outputs of the row groups meet in shared memory in a fixed order.
template <typename T>
__global__ void __launch_bounds__(256, 4) ssd_step_kernel(
    const T* __restrict__ x, long ldx, const T* __restrict__ b, long ldb, const T* __restrict__ c, long ldc,
    const T* __restrict__ dt, long lddt, const float* __restrict__ neg_a, const float* __restrict__ dt_bias,
    const float* __restrict__ d_skip, float* __restrict__ state, const int* __restrict__ rec_slots,
    const int* __restrict__ seq_lens, const int* __restrict__ qsl, int H, int G, int N, int V,
    float* __restrict__ out) {
  extern __shared__ float sm[];
  float* sb = sm;                 // [N]
  float* sc = sm + N;             // [N]
  float* part = sm + 2 * N;       // [row groups][V]
  const int h = blockIdx.x, s = blockIdx.y;
  const int q0 = qsl[s], n_tok = qsl[s + 1] - q0;
  if (n_tok <= 0) return;
  const int grp = h / (H / G), cols = V / 4, rg = 256 / cols;
  const int col = (threadIdx.x % cols) * 4, r0 = threadIdx.x / cols;
  const size_t t = q0;
  for (int i = threadIdx.x; i < N; i += 256) {
    sb[i] = to_f(b[t * ldb + (size_t)grp * N + i]);
    sc[i] = to_f(c[t * ldc + (size_t)grp * N + i]);
  }
  const float dtv = softplus_f(to_f(dt[t * lddt + h]) + dt_bias[h]);
  const float g = expf(neg_a[h] * dtv);
  const bool carried = state != nullptr && seq_lens[s] > n_tok;
  float* st = state != nullptr ? state + ((size_t)rec_slots[s] * H + h) * (size_t)N * V : nullptr;
  float xv[4], u[4];
  const bool on = r0 < rg;
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    xv[e] = to_f(x[t * ldx + (size_t)h * V + col + e]);
    u[e] = dtv * xv[e];
  }
  __syncthreads();
  float y[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) {
    constexpr int ROWS = 4;
    for (int n0 = r0; n0 < N; n0 += rg * ROWS) {
      float4 S[ROWS];
#pragma unroll
      for (int k = 0; k < ROWS; ++k) {
        const int n = n0 + k * rg;
        S[k] = (carried && n < N) ? __ldcs(reinterpret_cast<const float4*>(st + (size_t)n * V + col))
                                  : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int k = 0; k < ROWS; ++k) {
        const int n = n0 + k * rg;
        if (n < N) {
          const float bn = sb[n], cn = sc[n];
          S[k].x = fmaf(bn, u[0], g * S[k].x);
          S[k].y = fmaf(bn, u[1], g * S[k].y);
          S[k].z = fmaf(bn, u[2], g * S[k].z);
          S[k].w = fmaf(bn, u[3], g * S[k].w);
          y[0] = fmaf(S[k].x, cn, y[0]);
          y[1] = fmaf(S[k].y, cn, y[1]);
          y[2] = fmaf(S[k].z, cn, y[2]);
          y[3] = fmaf(S[k].w, cn, y[3]);
          if (st != nullptr) __stcs(reinterpret_cast<float4*>(st + (size_t)n * V + col), S[k]);
        }
      }
    }
    *reinterpret_cast<float4*>(part + (size_t)r0 * V + col) = make_float4(y[0], y[1], y[2], y[3]);
  }
  __syncthreads();
  if (r0 == 0) {
    float4 tot = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < rg; ++k) {
      const float4 p = *reinterpret_cast<const float4*>(part + (size_t)k * V + col);
      tot.x += p.x; tot.y += p.y; tot.z += p.z; tot.w += p.w;
    }
    const float ds = d_skip[h];
    tot.x = fmaf(ds, xv[0], tot.x); tot.y = fmaf(ds, xv[1], tot.y);
    tot.z = fmaf(ds, xv[2], tot.z); tot.w = fmaf(ds, xv[3], tot.w);
    *reinterpret_cast<float4*>(out + t * (size_t)H * V + (size_t)h * V + col) = tot;
  }
}

// ---------------------------------------------------------------------------------------------------------------
// Chunked form for longer portions (bf16 inputs). With the running sums L_t of the log decays inside a chunk of 64 tokens
//     y_t   = exp(L_t) C_t S_0 + sum_{j <= t} (C_t . B_j) exp(L_t - L_j) dt_j x_j + d x_t
//     S_end = exp(L_63) S_0 + sum_j B_j (exp(L_63 - L_j) dt_j x_j)^T
// so a chunk is four small matrix products on the tensor cores and only S is carried from chunk to chunk (in fp32
// accumulators). C, B and x are exact bf16; the fp32 operands (S, the weighted scores, the weighted x) are split into
// a bf16 head and a bf16 remainder and multiplied twice, which keeps 16 significant bits of each.
// One block per (sequence, head, VT value columns), NW = 4 or 8 warps: warp w works on tokens 16 (w % 4) .. + 15 of the
// chunk and on one of NW / 4 shares of the value columns in the output products, and on a share of the state rows (WM
// warps) and value columns (NW / WM) in the state update.
constexpr int kQ = 64;

__device__ __forceinline__ uint32_t s_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4_t(uint32_t a, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// head and remainder of two fp32 values as packed bf16 pairs
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 hf = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - hf.x, b - hf.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ void cp16(void* dst, const void* src, bool ok) {
  const int sz = ok ? 16 : 0;                     // 0: the 16 bytes are zero-filled, the source is not read
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s_addr(dst)), "l"(src), "r"(sz));
}

template <int NP, int VT>
struct SsdSmem {
  static constexpr int LN = NP + 8, LV = VT + 8;  // row strides (elements) that keep ldmatrix conflict-free
  static constexpr int B = 0, C = B + kQ * LN, X = C + kQ * LN, SH = X + kQ * LV, SL = SH + NP * LV,
                       WH = SL + NP * LV, WL = WH + kQ * LV, kElems = WL + kQ * LV;
  static constexpr int kBytes = kElems * 2 + 5 * kQ * 4;
};

template <int NP, int VT, int NW>
__global__ void __launch_bounds__(32 * NW, NW == 8 ? 2 : 1) ssd_chunk_kernel(
    const bf16_t* __restrict__ x, long ldx, const bf16_t* __restrict__ b, long ldb, const bf16_t* __restrict__ c,
    long ldc, const bf16_t* __restrict__ dt, long lddt, const float* __restrict__ neg_a,
    const float* __restrict__ dt_bias, const float* __restrict__ d_skip, float* __restrict__ state,
    const int* __restrict__ rec_slots, const int* __restrict__ seq_lens, const int* __restrict__ qsl, int H, int G,
    int N, int V, float* __restrict__ out) {
  using SM = SsdSmem<NP, VT>;
  constexpr int LN = SM::LN, LV = SM::LV;
  constexpr int NT = 32 * NW, CS = NW / 4, VC = VT / 8 / CS;   // column shares; 8-wide column tiles of a warp's share
  constexpr int MT = NP / 16, WM = MT < NW ? MT : NW, WN = NW / WM;
  constexpr int MI = MT / WM, NI = VT / 8 / WN;   // state tiles (16 x 8) of a warp
  static_assert(NI % 2 == 0 && VC % 2 == 0, "column tiles come in pairs");
  extern __shared__ __align__(16) uint8_t smem_raw[];
  bf16_t* sm = reinterpret_cast<bf16_t*>(smem_raw);
  bf16_t *sB = sm + SM::B, *sC = sm + SM::C, *sX = sm + SM::X, *sSh = sm + SM::SH, *sSl = sm + SM::SL,
         *sWh = sm + SM::WH, *sWl = sm + SM::WL;
  float* sLh = reinterpret_cast<float*>(sm + SM::kElems);   // running log decay: head, remainder
  float *sLl = sLh + kQ, *sDt = sLl + kQ, *sWt = sDt + kQ, *sEl = sWt + kQ;

  const int h = blockIdx.x, v0 = blockIdx.y * VT, s = blockIdx.z;
  const int q0 = qsl[s], q1 = qsl[s + 1];
  if (q1 <= q0) return;                           // uniform over the block
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g4 = lane >> 2, t4 = lane & 3, lq = lane >> 3, lr = lane & 7;
  const int grp = h / (H / G);
  const int wm = warp % WM, wn = warp / WM;
  const int tw = warp & 3, cb = (warp >> 2) * VC;    // output products: token group, first column tile
  const bool carried = state != nullptr && seq_lens[s] > q1 - q0;
  float* st = state != nullptr ? state + ((size_t)rec_slots[s] * H + h) * (size_t)N * V : nullptr;
  const float na = neg_a[h], db = dt_bias[h], ds = d_skip[h];
  const bf16_t* bp = b + (size_t)grp * N;
  const bf16_t* cp = c + (size_t)grp * N;
  const bf16_t* xp = x + (size_t)h * V + v0;

  float S[MI][NI][4];
#pragma unroll
  for (int mi = 0; mi < MI; ++mi)
#pragma unroll
    for (int ni = 0; ni < NI; ++ni)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = (wm * MI + mi) * 16 + g4 + 8 * (e >> 1), v = v0 + (wn * NI + ni) * 8 + 2 * t4 + (e & 1);
        S[mi][ni][e] = (carried && n < N && v < V) ? st[(size_t)n * V + v] : 0.f;
      }

  for (int t0 = q0; t0 < q1; t0 += kQ) {
    const int nt = min(kQ, q1 - t0);
    __syncthreads();                              // the previous chunk's tiles are consumed
    for (int i = threadIdx.x; i < kQ * (NP / 8); i += NT) {
      const int r = i / (NP / 8), e = (i % (NP / 8)) * 8;
      const bool ok = r < nt && e < N;
      const size_t row = t0 + (ok ? r : 0);
      cp16(sB + r * LN + e, bp + row * ldb + (ok ? e : 0), ok);
      cp16(sC + r * LN + e, cp + row * ldc + (ok ? e : 0), ok);
    }
    for (int i = threadIdx.x; i < kQ * (VT / 8); i += NT) {
      const int r = i / (VT / 8), e = (i % (VT / 8)) * 8;
      const bool ok = r < nt && v0 + e < V;
      const size_t row = t0 + (ok ? r : 0);
      cp16(sX + r * LV + e, xp + row * ldx + (ok ? e : 0), ok);
    }
    asm volatile("cp.async.commit_group;");
    // the state as it enters the chunk, split for the C . S product
#pragma unroll
    for (int mi = 0; mi < MI; ++mi)
#pragma unroll
      for (int ni = 0; ni < NI; ++ni)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int off = ((wm * MI + mi) * 16 + g4 + 8 * r) * LV + (wn * NI + ni) * 8 + 2 * t4;
          uint32_t hi, lo;
          split2(S[mi][ni][2 * r], S[mi][ni][2 * r + 1], hi, lo);
          *reinterpret_cast<uint32_t*>(sSh + off) = hi;
          *reinterpret_cast<uint32_t*>(sSl + off) = lo;
        }
    if (warp == 0) {                              // tokens 2 lane, 2 lane + 1: steps and running log decays
      float d0 = 0.f, d1 = 0.f;
      if (2 * lane < nt) d0 = softplus_f(to_f(dt[(size_t)(t0 + 2 * lane) * lddt + h]) + db);
      if (2 * lane + 1 < nt) d1 = softplus_f(to_f(dt[(size_t)(t0 + 2 * lane + 1) * lddt + h]) + db);
      const double a0 = (double)(na * d0), a1 = (double)(na * d1);
      double run = a0 + a1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
      }
      const double end = __shfl_sync(0xffffffffu, run, 31);
      const double l1 = run, l0 = run - a1;
      sLh[2 * lane] = (float)l0;
      sLl[2 * lane] = (float)(l0 - (double)(float)l0);
      sLh[2 * lane + 1] = (float)l1;
      sLl[2 * lane + 1] = (float)(l1 - (double)(float)l1);
      sDt[2 * lane] = d0;
      sDt[2 * lane + 1] = d1;
      sEl[2 * lane] = expf((float)l0);
      sEl[2 * lane + 1] = expf((float)l1);
      sWt[2 * lane] = expf((float)(end - l0)) * d0;
      sWt[2 * lane + 1] = expf((float)(end - l1)) * d1;
    }
    asm volatile("cp.async.wait_group 0;");
    __syncthreads();
    for (int i = threadIdx.x; i < kQ * (VT / 2); i += NT) {
      const int r = i / (VT / 2), e = (i % (VT / 2)) * 2;
      const float2 xv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sX + r * LV + e));
      const float w = sWt[r];
      uint32_t hi, lo;
      split2(w * xv.x, w * xv.y, hi, lo);
      *reinterpret_cast<uint32_t*>(sWh + r * LV + e) = hi;
      *reinterpret_cast<uint32_t*>(sWl + r * LV + e) = lo;
    }
    // ---- C . S (entering state) and C . B^T for this warp's 16 tokens
    float acc[VC][4], G2[8][4];
#pragma unroll
    for (int i = 0; i < VC; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) G2[i][0] = G2[i][1] = G2[i][2] = G2[i][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < NP / 16; ++ks) {
      uint32_t a[4];
      ldsm4(s_addr(sC + (tw * 16 + (lq & 1) * 8 + lr) * LN + ks * 16 + (lq >> 1) * 8), a);
#pragma unroll
      for (int nv = 0; nv < VC; nv += 2) {
        uint32_t r[4];
        const int off = (ks * 16 + (lq & 1) * 8 + lr) * LV + (cb + nv) * 8 + (lq >> 1) * 8;
        ldsm4_t(s_addr(sSh + off), r);
        mma16816(acc[nv], a, r[0], r[1]);
        mma16816(acc[nv + 1], a, r[2], r[3]);
        ldsm4_t(s_addr(sSl + off), r);
        mma16816(acc[nv], a, r[0], r[1]);
        mma16816(acc[nv + 1], a, r[2], r[3]);
      }
#pragma unroll
      for (int jt = 0; jt < 8; jt += 2) {
        if (jt <= 2 * tw) {                     // keys after the warp's last token are not needed
          uint32_t r[4];
          ldsm4(s_addr(sB + (jt * 8 + (lq >> 1) * 8 + lr) * LN + ks * 16 + (lq & 1) * 8), r);
          mma16816(G2[jt], a, r[0], r[1]);
          mma16816(G2[jt + 1], a, r[2], r[3]);
        }
      }
    }
    const int ta = tw * 16 + g4, tb = ta + 8;
    const float ea = sEl[ta], eb = sEl[tb];
#pragma unroll
    for (int i = 0; i < VC; ++i) { acc[i][0] *= ea; acc[i][1] *= ea; acc[i][2] *= eb; acc[i][3] *= eb; }
    // ---- weighted scores times x
    const float lha = sLh[ta], lla = sLl[ta], lhb = sLh[tb], llb = sLl[tb];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      if (kk <= tw) {
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          float p[4];
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int j = kk * 16 + half * 8 + 2 * t4 + e;
            const float lh = sLh[j], ll = sLl[j], d = sDt[j];
            p[e] = j <= ta ? G2[2 * kk + half][e] * (expf((lha - lh) + (lla - ll)) * d) : 0.f;
            p[2 + e] = j <= tb ? G2[2 * kk + half][2 + e] * (expf((lhb - lh) + (llb - ll)) * d) : 0.f;
          }
          split2(p[0], p[1], ph[2 * half], pl[2 * half]);
          split2(p[2], p[3], ph[2 * half + 1], pl[2 * half + 1]);
        }
#pragma unroll
        for (int nv = 0; nv < VC; nv += 2) {
          uint32_t r[4];
          ldsm4_t(s_addr(sX + (kk * 16 + (lq & 1) * 8 + lr) * LV + (cb + nv) * 8 + (lq >> 1) * 8), r);
          mma16816(acc[nv], ph, r[0], r[1]);
          mma16816(acc[nv + 1], ph, r[2], r[3]);
          mma16816(acc[nv], pl, r[0], r[1]);
          mma16816(acc[nv + 1], pl, r[2], r[3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < VC; ++i)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int tk = r == 0 ? ta : tb, vv = (cb + i) * 8 + 2 * t4;
        if (tk < nt && v0 + vv < V) {
          const float2 xv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sX + tk * LV + vv));
          *reinterpret_cast<float2*>(out + (size_t)(t0 + tk) * H * V + (size_t)h * V + v0 + vv) =
              make_float2(fmaf(ds, xv.x, acc[i][2 * r]), fmaf(ds, xv.y, acc[i][2 * r + 1]));
        }
      }
    __syncthreads();                              // the weighted x is complete
    // ---- state update
    const float ge = sEl[kQ - 1];
#pragma unroll
    for (int mi = 0; mi < MI; ++mi)
#pragma unroll
      for (int ni = 0; ni < NI; ++ni)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[mi][ni][e] *= ge;
#pragma unroll
    for (int ks = 0; ks < kQ / 16; ++ks) {
      uint32_t a[MI][4];
#pragma unroll
      for (int mi = 0; mi < MI; ++mi)
        ldsm4_t(s_addr(sB + (ks * 16 + (lq >> 1) * 8 + lr) * LN + (wm * MI + mi) * 16 + (lq & 1) * 8), a[mi]);
#pragma unroll
      for (int ni = 0; ni < NI; ni += 2) {
        uint32_t rh[4], rl[4];
        const int off = (ks * 16 + (lq & 1) * 8 + lr) * LV + (wn * NI + ni) * 8 + (lq >> 1) * 8;
        ldsm4_t(s_addr(sWh + off), rh);
        ldsm4_t(s_addr(sWl + off), rl);
#pragma unroll
        for (int mi = 0; mi < MI; ++mi) {
          mma16816(S[mi][ni], a[mi], rh[0], rh[1]);
          mma16816(S[mi][ni + 1], a[mi], rh[2], rh[3]);
          mma16816(S[mi][ni], a[mi], rl[0], rl[1]);
          mma16816(S[mi][ni + 1], a[mi], rl[2], rl[3]);
        }
      }
    }
  }
  if (st != nullptr) {
#pragma unroll
    for (int mi = 0; mi < MI; ++mi)
#pragma unroll
      for (int ni = 0; ni < NI; ++ni)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int n = (wm * MI + mi) * 16 + g4 + 8 * (e >> 1), v = v0 + (wn * NI + ni) * 8 + 2 * t4 + (e & 1);
          if (n < N && v < V) st[(size_t)n * V + v] = S[mi][ni][e];
        }
  }
}

template <int NP, int VT, int NW>
int launch_chunk(int nseq, cudaStream_t stm, const void* x, long ldx, const void* b, long ldb, const void* c, long ldc,
                 const void* dt, long lddt, const float* neg_a, const float* dt_bias, const float* d_skip, float* state,
                 const int* rec_slots, const int* seq_lens, const int* qsl, int H, int G, int N, int V, float* out) {
  using SM = SsdSmem<NP, VT>;
  CUDA_CHECK_RET(cudaFuncSetAttribute(ssd_chunk_kernel<NP, VT, NW>, cudaFuncAttributeMaxDynamicSharedMemorySize, SM::kBytes));
  dim3 grid(H, (V + VT - 1) / VT, nseq);
  ssd_chunk_kernel<NP, VT, NW><<<grid, 32 * NW, SM::kBytes, stm>>>(
      (const bf16_t*)x, ldx, (const bf16_t*)b, ldb, (const bf16_t*)c, ldc, (const bf16_t*)dt, lddt, neg_a, dt_bias,
      d_skip, state, rec_slots, seq_lens, qsl, H, G, N, V, out);
  CUDA_CHECK_RET(cudaGetLastError());
  return 0;
}

}  // namespace

#define GLLM_BY_DTYPE(is_f32, CALL_BF16, CALL_F32) \
  do { if (is_f32) { CALL_F32; } else { CALL_BF16; } } while (0)

GLLM_EXPORT int gllm_ssd_rotary_angles(const void* positions, const void* freqs, int n, void* out, int ntok,
                                       void* stream) {
  if (ntok <= 0 || n <= 0) return 0;
  const size_t total = (size_t)ntok * n;
  rotary_angles_kernel<<<(unsigned)((total + 127) / 128), 128, 0, (cudaStream_t)stream>>>(
      (const int*)positions, (const double*)freqs, n, (float*)out, total);
  CUDA_CHECK_RET(cudaGetLastError());
  return 0;
}

GLLM_EXPORT int gllm_ssd_gelu_gate_embed(const void* g, long ldg, const void* ids, int vocab, const void* table,
                                         long ldt, int col0, void* out, int ntok, int dim, int is_f32, void* stream) {
  if (ntok <= 0 || dim <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  const size_t total = (size_t)ntok * dim;
  const unsigned blocks = (unsigned)((total + 255) / 256);
  GLLM_BY_DTYPE(is_f32,
                (gelu_gate_embed_kernel<bf16_t><<<blocks, 256, 0, st>>>((const bf16_t*)g, ldg, (const int*)ids, vocab,
                                                                        (const bf16_t*)table, ldt, col0, (bf16_t*)out,
                                                                        dim, total)),
                (gelu_gate_embed_kernel<float><<<blocks, 256, 0, st>>>((const float*)g, ldg, (const int*)ids, vocab,
                                                                       (const float*)table, ldt, col0, (float*)out,
                                                                       dim, total)));
  CUDA_CHECK_RET(cudaGetLastError());
  return 0;
}

GLLM_EXPORT int gllm_ssd_gate_then_norm(const void* o, int n, const void* gate, long ldg, const void* w, int group,
                                        float eps, void* out, long ldo, int ntok, int is_f32, void* stream) {
  if (ntok <= 0 || n <= 0) return 0;
  if (group <= 0 || n % group != 0) return 2;
  cudaStream_t st = (cudaStream_t)stream;
  dim3 grid(ntok, n / group);
  if (!is_f32 && group % 4 == 0 && group <= 8192 && ldg % 4 == 0 && ldo % 4 == 0 && ((uintptr_t)gate & 7) == 0 &&
      ((uintptr_t)out & 7) == 0 && ((uintptr_t)o & 15) == 0 && ((uintptr_t)w & 15) == 0) {
    int threads = (group / 4 + 31) / 32 * 32;
    threads = threads > 256 ? 256 : threads;
    const int per = (group / 4 + threads - 1) / threads;
#define GLLM_GTN(MV)                                                                                              \
  gate_then_norm_vec_kernel<MV><<<grid, threads, 0, st>>>((const float*)o, n, (const bf16_t*)gate, ldg,           \
                                                          (const float*)w, group, eps, (bf16_t*)out, ldo)
    if (per <= 1) GLLM_GTN(1);
    else if (per <= 2) GLLM_GTN(2);
    else if (per <= 4) GLLM_GTN(4);
    else GLLM_GTN(8);
#undef GLLM_GTN
    CUDA_CHECK_RET(cudaGetLastError());
    return 0;
  }
  const size_t smem = (size_t)group * sizeof(float);
  if (smem > 200 * 1024) return 2;
  if (smem > 48 * 1024) {
    CUDA_CHECK_RET(cudaFuncSetAttribute(gate_then_norm_kernel<bf16_t>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                        200 * 1024));
    CUDA_CHECK_RET(cudaFuncSetAttribute(gate_then_norm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                        200 * 1024));
  }
  const int threads = group >= 256 ? 256 : (group + 31) / 32 * 32;
  GLLM_BY_DTYPE(is_f32,
                (gate_then_norm_kernel<bf16_t><<<grid, threads, smem, st>>>((const float*)o, n, (const bf16_t*)gate,
                                                                            ldg, (const float*)w, group, eps,
                                                                            (bf16_t*)out, ldo)),
                (gate_then_norm_kernel<float><<<grid, threads, smem, st>>>((const float*)o, n, (const float*)gate, ldg,
                                                                           (const float*)w, group, eps, (float*)out,
                                                                           ldo)));
  CUDA_CHECK_RET(cudaGetLastError());
  return 0;
}

// sequences of one token each: V % 4 == 0, V <= 1024, 16-byte aligned state; returns 2 outside that
GLLM_EXPORT int gllm_ssd_step(const void* x, long ldx, const void* b, long ldb, const void* c, long ldc, const void* dt,
                              long lddt, const void* neg_a, const void* dt_bias, const void* d_skip, void* state,
                              const void* rec_slots, const void* seq_lens, const void* qsl, int nseq, int H, int G,
                              int N, int V, void* out, int is_f32, void* stream) {
  if (nseq <= 0) return 0;
  if (V % 4 != 0 || V > 1024 || ((uintptr_t)state & 15) != 0 || ((uintptr_t)out & 15) != 0 || nseq > 65535) return 2;
  const int rg = 256 / (V / 4);
  const size_t smem = (size_t)(2 * N + rg * V) * sizeof(float);
  if (smem > 48 * 1024 || N % 2 != 0) return 2;
  cudaStream_t st = (cudaStream_t)stream;
  dim3 grid(H, nseq);
#define GLLM_STEP(T)                                                                                                 \
  ssd_step_kernel<T><<<grid, 256, smem, st>>>((const T*)x, ldx, (const T*)b, ldb, (const T*)c, ldc, (const T*)dt,   \
                                              lddt, (const float*)neg_a, (const float*)dt_bias,                     \
                                              (const float*)d_skip, (float*)state, (const int*)rec_slots,           \
                                              (const int*)seq_lens, (const int*)qsl, H, G, N, V, (float*)out)
  if (is_f32) GLLM_STEP(float);
  else GLLM_STEP(bf16_t);
#undef GLLM_STEP
  CUDA_CHECK_RET(cudaGetLastError());
  return 0;
}

// portions of any length, bf16: N <= 256, N % 8 == 0, V % 8 == 0, 16-byte aligned rows; returns 2 outside that
GLLM_EXPORT int gllm_ssd_chunk(const void* x, long ldx, const void* b, long ldb, const void* c, long ldc,
                               const void* dt, long lddt, const void* neg_a, const void* dt_bias, const void* d_skip,
                               void* state, const void* rec_slots, const void* seq_lens, const void* qsl, int nseq,
                               int H, int G, int N, int V, void* out, void* stream) {
  if (nseq <= 0) return 0;
  if (N > 256 || N % 8 != 0 || V % 8 != 0 || ldx % 8 != 0 || ldb % 8 != 0 || ldc % 8 != 0 || nseq > 65535 ||
      ((uintptr_t)x & 15) != 0 || ((uintptr_t)b & 15) != 0 || ((uintptr_t)c & 15) != 0 || ((uintptr_t)out & 7) != 0)
    return 2;
  cudaStream_t st = (cudaStream_t)stream;
#define GLLM_CHUNK(NP, VT, NW)                                                                                          \
  return launch_chunk<NP, VT, NW>(nseq, st, x, ldx, b, ldb, c, ldc, dt, lddt, (const float*)neg_a, (const float*)dt_bias, \
                              (const float*)d_skip, (float*)state, (const int*)rec_slots, (const int*)seq_lens,      \
                              (const int*)qsl, H, G, N, V, (float*)out)
  // narrower column blocks where 64-wide ones leave SMs idle (every column is computed alike in both)
  const bool narrow = V <= 32 || (long)H * nseq * ((V + 63) / 64) <= 148;
  if (N <= 32) { if (narrow) GLLM_CHUNK(32, 32, 4); else GLLM_CHUNK(32, 64, 8); }
  if (N <= 64) { if (narrow) GLLM_CHUNK(64, 32, 8); else GLLM_CHUNK(64, 64, 8); }
  if (N <= 128) { if (narrow) GLLM_CHUNK(128, 32, 8); else GLLM_CHUNK(128, 64, 8); }
  GLLM_CHUNK(256, 32, 8);
#undef GLLM_CHUNK
}

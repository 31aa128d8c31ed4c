// k_stack_delta.cu -- the gated delta rule of the layer-list decoders (DIS_MIX_CHANNEL_DELTA): short convolutions, unit lengths,
// decays and step sizes of the pass's tokens, and the recurrence itself over a per-slot state.  Everything that enters the
// recurrence is fp32, and so is the state.
#include <algorithm>
#include "stack_dev.cuh"

namespace dis {

// ------------------------------------------------------------------------------------------------ preparation
// One launch; blockIdx.x is a tile of tokens, blockIdx.y a role:
//   [0, G)            queries and keys of one key head: convolution, SiLU, division by the length (queries also times d^(-1/2)),
//                     and their inner product
//   then nvb blocks   128 value channels each: convolution and SiLU (the first also forms the step sizes sigmoid(.))
//   then ndb blocks   128 decays each: exp(-exp(A_log) softplus(z + dt_bias)), z from memory or as the product with the bottleneck
//   then ngb blocks   128 logits of the output gate each, as products with their bottleneck (absent when z comes from memory)
// The input projection may come as n_part split-K slices, summed where they are read.
constexpr int kDeltaTh = 128, kDeltaMaxTaps = 16;
__device__ __forceinline__ float delta_silu(float v) { return v / (1.f + expf(-v)); }

// sum_r w[row][r] u[r] over a bottleneck; u in shared memory (16-byte aligned)
template <bool WF32>
__device__ __forceinline__ float delta_row_dot(const void *w, long long row, const float *u, int n) {
  float s0 = 0.f, s1 = 0.f;
  if ((n & 7) == 0) {
    for (int r = 0; r < n; r += 8) {
      float wv[8];
      if (WF32) {
        const float4 a = *reinterpret_cast<const float4 *>(reinterpret_cast<const float *>(w) + row * n + r);
        const float4 b = *reinterpret_cast<const float4 *>(reinterpret_cast<const float *>(w) + row * n + r + 4);
        wv[0] = a.x; wv[1] = a.y; wv[2] = a.z; wv[3] = a.w; wv[4] = b.x; wv[5] = b.y; wv[6] = b.z; wv[7] = b.w;
      } else {
        const uint4 v = *reinterpret_cast<const uint4 *>(reinterpret_cast<const uint16_t *>(w) + row * n + r);
        const uint32_t q[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int j = 0; j < 4; j++) { wv[2 * j] = __uint_as_float(q[j] << 16); wv[2 * j + 1] = __uint_as_float(q[j] & 0xffff0000u); }
      }
      const float4 ua = *reinterpret_cast<const float4 *>(u + r), ub = *reinterpret_cast<const float4 *>(u + r + 4);
      s0 = fmaf(wv[0], ua.x, s0); s1 = fmaf(wv[1], ua.y, s1); s0 = fmaf(wv[2], ua.z, s0); s1 = fmaf(wv[3], ua.w, s1);
      s0 = fmaf(wv[4], ub.x, s0); s1 = fmaf(wv[5], ub.y, s1); s0 = fmaf(wv[6], ub.z, s0); s1 = fmaf(wv[7], ub.w, s1);
    }
  } else
    for (int r = 0; r < n; r++) s0 = fmaf(ld_el<WF32>(w, row * n + r), u[r], s0);
  return s0 + s1;
}

// TAPS 1 .. 4: the convolution's window sits in registers; 0: any number of taps, every input read again for every token that needs
// it.  The input at position p comes from the span's rows or, before the span, from the slot's tail (tail[i] holds position pos0 -
// (taps - 1) + i); before the sequence's start it is zero, so a slot that was used before needs no clearing.  single: every span
// is one token, and its thread moves the tail on itself.
template <int TAPS, bool WF32>
__global__ void __launch_bounds__(kDeltaTh) stack_delta_prep_kernel(StackDelta c, StackDeltaPrep a, StackSpans sp, int tile, int nvb, int ndb, int single) {
  extern __shared__ __align__(16) float sh[];
  const int t0 = blockIdx.x * tile, t1 = min(sp.T, t0 + tile);
  const int taps = TAPS ? TAPS : c.taps, C = c.C;
  auto in = [&](int t, int col) {
    const float *p = a.proj + (long long)t * a.ld + col;
    float v = p[0];
    for (int k = 1; k < a.n_part; k++) v += p[(long long)k * a.stride];
    return v;
  };
  auto conv = [&](int ch, auto &&put) {  // channel ch of q | k | v over the tile's tokens
    constexpr int TW = TAPS > 1 ? TAPS - 1 : 1;
    float w[TAPS ? TAPS : 1], win[TW];
    if (TAPS) {
#pragma unroll
      for (int j = 0; j < (TAPS ? TAPS : 1); j++) w[j] = a.cw[(long long)ch * taps + j];
    }
    int prev = -1;
    constexpr int U = 8;
    for (int tb = t0; tb < t1; tb += U) {
      float cur[U];
#pragma unroll
      for (int u = 0; u < U; u++) cur[u] = tb + u < t1 ? in(tb + u, ch) : 0.f;
#pragma unroll
      for (int u = 0; u < U; u++) {
        const int t = tb + u;
        if (t >= t1) break;
        const int s = sp.span[t];
        const int back_in_span = t - sp.sp_tok0[s], pos0 = sp.sp_pos0[s];
        float *tail = a.cstate + (long long)sp.sp_slot[s] * (taps - 1) * C + ch;
        auto before = [&](int back) {  // the input `back` tokens before t
          if (back <= back_in_span) return in(t - back, ch);
          return pos0 + back_in_span - back >= 0 ? tail[(long long)((taps - 1) - (back - back_in_span)) * C] : 0.f;
        };
        float acc = 0.f;
        if (TAPS) {
          if (s != prev) {
            prev = s;
#pragma unroll
            for (int j = 0; j < TW; j++) win[j] = TAPS > 1 ? before(taps - 1 - j) : 0.f;
          }
#pragma unroll
          for (int j = 0; j + 1 < (TAPS ? TAPS : 1); j++) acc = fmaf(w[j], win[j], acc);
          acc = fmaf(w[TAPS ? TAPS - 1 : 0], cur[u], acc);
#pragma unroll
          for (int j = 0; j + 1 < TW; j++) win[j] = win[j + 1];
          if (TAPS > 1) win[TW - 1] = cur[u];
          if (single && TAPS > 1) {
#pragma unroll
            for (int j = 0; j < TW; j++) tail[(long long)j * C] = win[j];
          }
        } else {
          float old[kDeltaMaxTaps];
          for (int j = 0; j + 1 < taps; j++) {
            old[j] = before(taps - 1 - j);
            acc = fmaf(a.cw[(long long)ch * taps + j], old[j], acc);
          }
          acc = fmaf(a.cw[(long long)ch * taps + taps - 1], cur[u], acc);
          if (single) {
            for (int j = 0; j + 2 < taps; j++) tail[(long long)j * C] = old[j + 1];
            tail[(long long)(taps - 2) * C] = cur[u];
          }
        }
        put(t, delta_silu(acc));
      }
    }
  };
  int role = blockIdx.y;
  if (role < c.G) {
    const int g = role, d = c.d;
    float *qs = sh, *ks = sh + tile * d;
    for (int i = threadIdx.x; i < d; i += kDeltaTh) {
      conv(g * d + i, [&](int t, float v) { qs[(t - t0) * d + i] = v; });
      conv((c.G + g) * d + i, [&](int t, float v) { ks[(t - t0) * d + i] = v; });
    }
    __syncthreads();
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
    const float qscale = rsqrtf((float)d);
    for (int t = t0 + w; t < t1; t += kDeltaTh / 32) {
      const float *q = qs + (t - t0) * d, *k = ks + (t - t0) * d;
      float qq = 0.f, kk = 0.f, qk = 0.f;
      for (int i = l; i < d; i += 32) { qq = fmaf(q[i], q[i], qq); kk = fmaf(k[i], k[i], kk); qk = fmaf(q[i], k[i], qk); }
      qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
      const float rq = rsqrtf(qq + 1e-6f) * qscale, rk = rsqrtf(kk + 1e-6f);
      float *row = a.buf + (long long)t * a.ld_b;
      for (int i = l; i < d; i += 32) { row[g * d + i] = q[i] * rq; row[(c.G + g) * d + i] = k[i] * rk; }
      if (l == 0) row[C + g] = qk * rq * rk;
    }
    return;
  }
  role -= c.G;
  if (role < nvb) {
    const int ch = 2 * c.G * c.d + role * kDeltaTh + threadIdx.x;
    if (role == 0)
      for (int e = threadIdx.x; e < (t1 - t0) * c.H; e += kDeltaTh) {
        const int t = t0 + e / c.H, h = e % c.H;
        a.buf[(long long)t * a.ld_b + C + c.G + h] = sigmoid_precise(in(t, c.b_off + h));
      }
    if (ch < C) conv(ch, [&](int t, float v) { a.buf[(long long)t * a.ld_b + ch] = v; });
    return;
  }
  role -= nvb;
  const bool dec = role < ndb;
  if (!dec) role -= ndb;
  const int n = dec ? c.H * c.d : c.H * c.dv, i = role * kDeltaTh + threadIdx.x;
  const int rank = dec ? c.ra : c.rg, off = dec ? c.a_off : c.g_off, pitch = (rank + 3) & ~3;
  if (!a.z) {  // the tile's bottleneck values
    for (int e = threadIdx.x; e < (t1 - t0) * rank; e += kDeltaTh) {
      const int tt = e / rank, r = e - tt * rank;
      sh[tt * pitch + r] = in(t0 + tt, off + r);
    }
    __syncthreads();
  }
  if (i >= n) return;
  if (!dec) {
    for (int t = t0; t < t1; t++) a.gz[(long long)t * n + i] = delta_row_dot<WF32>(a.g2, i, sh + (t - t0) * pitch, rank);
    return;
  }
  const float ea = expf(a.vec[i / c.d]), bias = a.vec[c.H + i];
#pragma unroll 4
  for (int t = t0; t < t1; t++) {
    const float z = (a.z ? a.z[(long long)t * n + i] : delta_row_dot<WF32>(a.a2, i, sh + (t - t0) * pitch, rank)) + bias;
    const float spl = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
    a.dec[(long long)t * n + i] = expf(-ea * spl);
  }
}
cudaError_t launch_stack_delta_prep(const StackDelta &c, const StackDeltaPrep &a, bool w_f32, const StackSpans &sp, cudaStream_t st) {
  if (sp.T <= 0) return cudaSuccess;
  if (c.taps < 1 || c.taps > kDeltaMaxTaps) return cudaErrorInvalidValue;
  const int single = sp.T == sp.n_spans ? 1 : 0, tile = single ? 1 : 16;
  const int nvb = (c.H * c.dv + kDeltaTh - 1) / kDeltaTh, ndb = (c.H * c.d + kDeltaTh - 1) / kDeltaTh, ngb = a.z ? 0 : (c.H * c.dv + kDeltaTh - 1) / kDeltaTh;
  const int rank = std::max(c.ra, c.rg);
  const size_t shb = (size_t)tile * std::max(2 * c.d, a.z ? 0 : (rank + 3) & ~3) * sizeof(float);
  if (shb > 200 * 1024) return cudaErrorInvalidValue;
  const dim3 grid((sp.T + tile - 1) / tile, c.G + nvb + ndb + ngb);
#define DIS_DELTA_PREP(TP, F)                                                                                                                            \
  do {                                                                                                                                                  \
    static DeviceOnce once;                                                                                                                             \
    DIS_CUDA_TRY(once.run([&] { return cudaFuncSetAttribute(stack_delta_prep_kernel<TP, F>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); })); \
    stack_delta_prep_kernel<TP, F><<<grid, kDeltaTh, shb, st>>>(c, a, sp, tile, nvb, ndb, single);                                                      \
  } while (0)
#define DIS_DELTA_PREP_T(F)                                                                                                                              \
  do {                                                                                                                                                  \
    switch (c.taps) {                                                                                                                                   \
      case 1: DIS_DELTA_PREP(1, F); break;                                                                                                              \
      case 2: DIS_DELTA_PREP(2, F); break;                                                                                                              \
      case 3: DIS_DELTA_PREP(3, F); break;                                                                                                              \
      case 4: DIS_DELTA_PREP(4, F); break;                                                                                                              \
      default: DIS_DELTA_PREP(0, F);                                                                                                                    \
    }                                                                                                                                                   \
  } while (0)
  if (w_f32) DIS_DELTA_PREP_T(true);
  else DIS_DELTA_PREP_T(false);
#undef DIS_DELTA_PREP_T
#undef DIS_DELTA_PREP
  DIS_CUDA_TRY(cudaGetLastError());
  if (c.taps > 1 && !single) return launch_stack_conv_tail(a.proj, a.ld, a.n_part, a.stride, 0, a.cstate, sp, c.C, c.taps, st);
  return cudaSuccess;
}

// bottleneck columns of the projection (slices summed) -> contiguous rows in the compute type, the operands of the products with a2, g2
template <bool F32>
__global__ void stack_delta_pack_kernel(const float *proj, long long ld, int n_part, long long stride, int a_off, int ra, int g_off, int rg,
                                        void *ua, void *ug) {
  const long long t = blockIdx.x;
  for (int i = threadIdx.x; i < ra + rg; i += blockDim.x) {
    const float *p = proj + t * ld + (i < ra ? a_off + i : g_off + i - ra);
    float v = p[0];
    for (int k = 1; k < n_part; k++) v += p[(long long)k * stride];
    if (i < ra) st_el<F32>(ua, t * ra + i, v);
    else st_el<F32>(ug, t * rg + i - ra, v);
  }
}
cudaError_t launch_stack_delta_pack(const StackDelta &c, const StackDeltaPrep &a, bool f32, int T, void *ua, void *ug, cudaStream_t st) {
  if (T <= 0) return cudaSuccess;
  if (f32) stack_delta_pack_kernel<true><<<T, 128, 0, st>>>(a.proj, a.ld, a.n_part, a.stride, c.a_off, c.ra, c.g_off, c.rg, ua, ug);
  else stack_delta_pack_kernel<false><<<T, 128, 0, st>>>(a.proj, a.ld, a.n_part, a.stride, c.a_off, c.ra, c.g_off, c.rg, ua, ug);
  return cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------ the recurrence
// Per head, S [d][dv]:  S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.
// The columns of S do not touch each other, so a head is cut into blocks of columns that never exchange anything: a warp owns 2 CL
// columns, its half-warps CL each, and the sixteen lanes of a half share the rows (RL each).  Both inner products run over the
// decayed state before the write -- o = (gS)^T q + u (k.q) -- so a token costs one reduction over sixteen lanes: a butterfly that
// halves the values a lane still carries at every step (products with k end in lanes 0-7, those with q in lanes 8-15), then u is
// handed back to all lanes.  Rows are taken in pairs by packed fp32 operations.  q, k, g, v, beta and k.q of the next kDeltaTok
// tokens are on their way into shared memory while the present ones are worked on; a CTA's warps share them.
// State: [slots][H][dv][d], a column's rows next to each other.
// fin.act: the CTA holds whole heads, and each token's o of the head is divided by its root mean square, times norm, times
// sigmoid(gate), and stored in the compute type; else o goes to o [T][H*dv] as it is.
constexpr int kDeltaTok = 8;
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) { f32x2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi)); return r; }
__device__ __forceinline__ void unpack2(f32x2 v, float &lo, float &hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) { f32x2 r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) { f32x2 r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }
__device__ __forceinline__ void delta_cp16(void *dst, const void *src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}
__device__ __forceinline__ void delta_cp4(void *dst, const void *src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

struct DeltaFin {
  void *act;
  long long ld;
  const float *gate;  // [T][H*dv]
  const float *norm;  // [dv]
  float eps;
  int f32;
};
template <int RL, int CL>
__global__ void __launch_bounds__(256, 1) stack_delta_kernel(StackDelta c, const float *__restrict__ buf, long long ld_b, const float *__restrict__ dec,
                                                          float *state, StackSpans sp, float *__restrict__ o, int ncb, int vec, DeltaFin fin) {
  extern __shared__ __align__(16) float sh[];
  constexpr int DP = 16 * RL, V = RL < 4 ? RL : 4, NM = RL / V, NP = RL / 2, CW = 2 * CL;
  const int H = c.H, d = c.d, dv = c.dv;
  const int h = blockIdx.x % H, rest = blockIdx.x / H, cb = rest % ncb, s = rest / ncb;  // heads vary fastest: CTAs that run together read whole rows
  const int tok0 = sp.sp_tok0[s], n = sp.sp_len[s], pos0 = sp.sp_pos0[s], slot = sp.sp_slot[s];
  const int NW = blockDim.x >> 5, w = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane & 15, hf = lane >> 4;
  const int VC = NW * CW, col_cta = cb * VC, nv = min(VC, dv - col_cta);
  const int PT = 3 * DP + VC + 4;  // a token's stage: q | k | g | v | beta, k.q
  float *os = sh + 2 * kDeltaTok * PT;  // [kDeltaTok][VC] outputs of a group (fin)
  for (int i = threadIdx.x; i < 2 * kDeltaTok * PT + (fin.act ? kDeltaTok * VC : 0); i += blockDim.x) sh[i] = 0.f;  // rows beyond d and columns beyond dv stay zero
  const int kvh = h / (H / c.G);
  const float *qsrc = buf + kvh * d, *ksrc = buf + (c.G + kvh) * d, *vsrc = buf + 2 * c.G * d + (long long)h * dv + col_cta;
  const float *gsrc = dec + (long long)h * d, *bsrc = buf + c.C + c.G + h, *xsrc = buf + c.C + kvh;
  auto fetch = [&](int i0, int stage) {
    const int ct = min(kDeltaTok, n - i0);
    float *dst0 = sh + stage * kDeltaTok * PT;
    const int per = vec ? 4 : 1, dq = d / per, nc = 3 * dq + nv / per;
    for (int i = threadIdx.x; i < ct * nc; i += blockDim.x) {
      const int tt = i / nc, e = i - tt * nc;
      const long long t = tok0 + i0 + tt;
      float *dst = dst0 + tt * PT;
      const float *src;
      if (e < dq) { src = qsrc + t * ld_b + e * per; dst += e * per; }
      else if (e < 2 * dq) { src = ksrc + t * ld_b + (e - dq) * per; dst += DP + (e - dq) * per; }
      else if (e < 3 * dq) { src = gsrc + t * (long long)H * d + (e - 2 * dq) * per; dst += 2 * DP + (e - 2 * dq) * per; }
      else { src = vsrc + t * ld_b + (e - 3 * dq) * per; dst += 3 * DP + (e - 3 * dq) * per; }
      if (vec) delta_cp16(dst, src);
      else delta_cp4(dst, src);
    }
    for (int i = threadIdx.x; i < 2 * ct; i += blockDim.x) {
      const long long t = tok0 + i0 + (i >> 1);
      delta_cp4(dst0 + (i >> 1) * PT + 3 * DP + VC + (i & 1), (i & 1 ? xsrc : bsrc) + t * ld_b);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // ---- the state: columns col0 + cc, rows r V + 16 V m + e
  const int wc = w * CW + hf * CL, col0 = col_cta + wc;
  float *st = state + ((long long)slot * H + h) * dv * d;
  f32x2 S[CL][NP];
#pragma unroll
  for (int cc = 0; cc < CL; cc++) {
    float v[RL];
    const float *p = st + (long long)(col0 + cc) * d;
    const bool on = pos0 > 0 && col0 + cc < dv;
#pragma unroll
    for (int m = 0; m < NM; m++) {
      const int i = r * V + 16 * V * m;
      if (V == 4 && vec) {
        const float4 f = on && i < d ? *reinterpret_cast<const float4 *>(p + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        v[m * V] = f.x; v[m * V + 1] = f.y; v[m * V + (V > 2 ? 2 : 0)] = f.z; v[m * V + (V > 3 ? 3 : 1)] = f.w;
      } else {
#pragma unroll
        for (int e = 0; e < V; e++) v[m * V + e] = on && i + e < d ? p[i + e] : 0.f;
      }
    }
#pragma unroll
    for (int q = 0; q < NP; q++) S[cc][q] = pack2(v[2 * q], v[2 * q + 1]);
  }
  __syncthreads();
  fetch(0, 0);
  const bool b3 = lane & 8, b2 = lane & 4, b1 = lane & 2, b0 = lane & 1;
  const int mycol = CL == 8 ? (lane & 7) : (lane & 7) >> 1;  // the column whose sums end in this lane
  int stage = 0;
  for (int i0 = 0; i0 < n; i0 += kDeltaTok, stage ^= 1) {
    const int ct = min(kDeltaTok, n - i0);
    if (i0 + kDeltaTok < n) {
      fetch(i0 + kDeltaTok, stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    for (int tt = 0; tt < ct; tt++) {
      const float *row = sh + (stage * kDeltaTok + tt) * PT;
      f32x2 kp[NP], qp[NP], gp[NP];
#pragma unroll
      for (int m = 0; m < NM; m++) {
        const float *p = row + r * V + 16 * V * m;
        if (V == 4) {
          const ulonglong2 a = *reinterpret_cast<const ulonglong2 *>(p), b = *reinterpret_cast<const ulonglong2 *>(p + DP), g = *reinterpret_cast<const ulonglong2 *>(p + 2 * DP);
          qp[2 * m] = a.x; qp[V == 4 ? 2 * m + 1 : 0] = a.y; kp[2 * m] = b.x; kp[V == 4 ? 2 * m + 1 : 0] = b.y; gp[2 * m] = g.x; gp[V == 4 ? 2 * m + 1 : 0] = g.y;
        } else {
          qp[m] = *reinterpret_cast<const f32x2 *>(p); kp[m] = *reinterpret_cast<const f32x2 *>(p + DP); gp[m] = *reinterpret_cast<const f32x2 *>(p + 2 * DP);
        }
      }
      const float vv = row[3 * DP + wc + mycol], beta = row[3 * DP + VC], kq = row[3 * DP + VC + 1];
      float x[CL];
#pragma unroll
      for (int cc = 0; cc < CL; cc++) {
        f32x2 a = 0ull, b = 0ull;
#pragma unroll
        for (int q = 0; q < NP; q++) {
          S[cc][q] = mul2(S[cc][q], gp[q]);
          a = fma2(S[cc][q], kp[q], a);
          b = fma2(S[cc][q], qp[q], b);
        }
        float al, ah, bl, bh;
        unpack2(a, al, ah); unpack2(b, bl, bh);
        const float dk = al + ah, dq = bl + bh;
        x[cc] = (b3 ? dq : dk) + __shfl_xor_sync(0xffffffffu, b3 ? dk : dq, 8);
      }
#pragma unroll
      for (int i = 0; i < CL / 2; i++) x[i] = (b2 ? x[i + CL / 2] : x[i]) + __shfl_xor_sync(0xffffffffu, b2 ? x[i] : x[i + CL / 2], 4);
#pragma unroll
      for (int i = 0; i < CL / 4; i++) x[i] = (b1 ? x[i + CL / 4] : x[i]) + __shfl_xor_sync(0xffffffffu, b1 ? x[i] : x[i + CL / 4], 2);
      if (CL == 8) x[0] = (b0 ? x[1] : x[0]) + __shfl_xor_sync(0xffffffffu, b0 ? x[0] : x[1], 1);
      else x[0] += __shfl_xor_sync(0xffffffffu, x[0], 1);
      const float u = beta * (vv - x[0]);  // (lanes 0-7 of a half)
#pragma unroll
      for (int cc = 0; cc < CL; cc++) {
        const float uc = __shfl_sync(0xffffffffu, u, (lane & 16) | (CL == 8 ? cc : 2 * cc));
        const f32x2 u2 = pack2(uc, uc);
#pragma unroll
        for (int q = 0; q < NP; q++) S[cc][q] = fma2(kp[q], u2, S[cc][q]);
      }
      const float ov = fmaf(__shfl_xor_sync(0xffffffffu, u, 8), kq, x[0]);  // (lanes 8-15)
      if (b3 && (CL == 8 || !b0)) {
        if (fin.act) os[tt * VC + wc + mycol] = ov;
        else if (col0 + mycol < dv) o[(long long)(tok0 + i0 + tt) * H * dv + (long long)h * dv + col0 + mycol] = ov;
      }
    }
    __syncthreads();
    if (fin.act) {  // a warp finishes a token (columns beyond dv are zero)
      for (int tt = w; tt < ct; tt += NW) {
        const float *ro = os + tt * VC;
        float ss = 0.f;
        for (int j = lane; j < dv; j += 32) ss = fmaf(ro[j], ro[j], ss);
        const float k = rsqrtf(warp_sum(ss) / (float)dv + fin.eps);
        const long long t = tok0 + i0 + tt;
        for (int j = lane; j < dv; j += 32) {
          const float v = ro[j] * k * fin.norm[j] * sigmoid_precise(fin.gate[t * H * dv + (long long)h * dv + j]);
          if (fin.f32) st_el<true>(fin.act, t * fin.ld + (long long)h * dv + j, v);
          else st_el<false>(fin.act, t * fin.ld + (long long)h * dv + j, v);
        }
      }
      if (i0 + kDeltaTok < n) __syncthreads();
    }
  }
#pragma unroll
  for (int cc = 0; cc < CL; cc++) {
    if (col0 + cc >= dv) continue;
    float *p = st + (long long)(col0 + cc) * d;
    float v[RL];
#pragma unroll
    for (int q = 0; q < NP; q++) unpack2(S[cc][q], v[2 * q], v[2 * q + 1]);
#pragma unroll
    for (int m = 0; m < NM; m++) {
      const int i = r * V + 16 * V * m;
      if (V == 4 && vec) {
        if (i < d) *reinterpret_cast<float4 *>(p + i) = make_float4(v[m * V], v[m * V + 1], v[m * V + (V > 2 ? 2 : 0)], v[m * V + (V > 3 ? 3 : 1)]);
      } else {
#pragma unroll
        for (int e = 0; e < V; e++)
          if (i + e < d) p[i + e] = v[m * V + e];
      }
    }
  }
}

template <int RL, int CL>
static cudaError_t delta_go(const StackDelta &c, const float *buf, long long ld_b, const float *dec, float *state, const StackSpans &sp, float *o,
                            int max_len, const float *norm, const float *gate, void *act, long long ld_act, bool f32, uint64_t *launches,
                            cudaStream_t st) {
  constexpr int CW = 2 * CL;
  const int total = (c.dv + CW - 1) / CW;  // warps that hold a head
  int nw = std::min(total, 8);
  // long spans: a head's columns are spread over more CTAs while that still brings idle SMs to work
  const long long pairs = (long long)sp.n_spans * c.H;
  while (max_len > kDeltaTok && nw > 2 && pairs * ((total + nw - 1) / nw) * 2 <= 148) nw = (nw + 1) / 2;
  const int ncb = (total + nw - 1) / nw, VC = nw * CW;
  const DeltaFin fin{ncb == 1 ? act : nullptr, ld_act, gate, norm, c.eps, f32 ? 1 : 0};
  auto al = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const int vec = c.d % 4 == 0 && c.dv % 4 == 0 && ld_b % 4 == 0 && al(buf) && al(dec) && al(state);
  const size_t shb = ((size_t)2 * kDeltaTok * (3 * 16 * RL + VC + 4) + (fin.act ? (size_t)kDeltaTok * VC : 0)) * sizeof(float);
  static DeviceOnce once;
  DIS_CUDA_TRY(once.run([&] { return cudaFuncSetAttribute(stack_delta_kernel<RL, CL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024); }));
  stack_delta_kernel<RL, CL><<<(unsigned)(pairs * ncb), nw * 32, shb, st>>>(c, buf, ld_b, dec, state, sp, o, ncb, vec, fin);
  DIS_CUDA_TRY(cudaGetLastError());
  *launches += fin.act ? 1 : 2;
  return fin.act ? cudaSuccess : launch_stack_headnorm_silu(o, norm, gate, (long long)c.H * c.dv, act, ld_act, 0, 1.f, f32, sp.T, c.H, c.dv, c.eps, st, true);
}
cudaError_t launch_stack_delta(const StackDelta &c, const float *buf, long long ld_b, const float *dec, float *state, const StackSpans &sp, float *o,
                               int max_len, const float *norm, const float *gate, void *act, long long ld_act, bool f32, uint64_t *launches, cudaStream_t st) {
#define DIS_DELTA(RL, CL) return delta_go<RL, CL>(c, buf, ld_b, dec, state, sp, o, max_len, norm, gate, act, ld_act, f32, launches, st)
  if (sp.T <= 0) return cudaSuccess;
  if (c.d <= 32) DIS_DELTA(2, 8);
  if (c.d <= 64) DIS_DELTA(4, 8);
  if (c.d <= 128) DIS_DELTA(8, 8);
  if (c.d <= 256) DIS_DELTA(16, 4);
#undef DIS_DELTA
  return cudaErrorInvalidValue;
}

}  // namespace dis

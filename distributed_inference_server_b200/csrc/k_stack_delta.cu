// k_stack_delta.cu -- the gated delta rule of the layer-list decoders (DIS_MIX_CHANNEL_DELTA): short convolutions, unit lengths,
// decays and step sizes of the pass's tokens, and the recurrence itself over a per-slot state.  Everything that enters the
// recurrence is fp32, and so is the state.
#include <algorithm>
#include "stack_dev.cuh"

namespace dis {

// ------------------------------------------------------------------------------------------------ preparation
// One launch; blockIdx.x is a tile of tokens, blockIdx.y a role:
//   [0, G)            queries and keys of one key head: convolution, SiLU, division by the length (queries also times d^(-1/2))
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
      float qq = 0.f, kk = 0.f;
      for (int i = l; i < d; i += 32) { qq = fmaf(q[i], q[i], qq); kk = fmaf(k[i], k[i], kk); }
      qq = warp_sum(qq); kk = warp_sum(kk);
      const float rq = rsqrtf(qq + 1e-6f) * qscale, rk = rsqrtf(kk + 1e-6f);
      float *row = a.buf + (long long)t * a.ld_b;
      for (int i = l; i < d; i += 32) { row[g * d + i] = q[i] * rq; row[(c.G + g) * d + i] = k[i] * rk; }
    }
    return;
  }
  role -= c.G;
  if (role < nvb) {
    const int ch = 2 * c.G * c.d + role * kDeltaTh + threadIdx.x;
    if (role == 0)
      for (int e = threadIdx.x; e < (t1 - t0) * c.H; e += kDeltaTh) {
        const int t = t0 + e / c.H, h = e % c.H;
        a.buf[(long long)t * a.ld_b + C + c.H * c.d + h] = sigmoid_precise(in(t, c.b_off + h));
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
    a.buf[(long long)t * a.ld_b + C + i] = expf(-ea * spl);
  }
}
// The same for passes with prompts whose sizes let a lane take four neighbouring channels (d and dv multiples of 4, d <= 128, decay
// logits from memory): a warp works on eight consecutive tokens and 128 channels by itself -- all their inputs are in flight together,
// and a head's squares are added up across the warp.  Roles as above, without the gate's.
constexpr int kDeltaWarpTok = 8, kDeltaVecTile = kDeltaWarpTok * kDeltaTh / 32;
template <int TAPS>
__global__ void __launch_bounds__(kDeltaTh, 4) stack_delta_prep_vec_kernel(StackDelta c, StackDeltaPrep a, StackSpans sp, int nvb) {
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, C = c.C;
  const int t0 = blockIdx.x * kDeltaVecTile + w * kDeltaWarpTok, nt = min(kDeltaWarpTok, sp.T - t0);
  if (nt <= 0) return;
  auto f4 = [](const float *p) { return *reinterpret_cast<const float4 *>(p); };
  auto in4 = [&](int t, int col) {
    const float *p = a.proj + (long long)t * a.ld + col;
    float4 v = f4(p);
    for (int k = 1; k < a.n_part; k++) {
      const float4 q = f4(p + (long long)k * a.stride);
      v.x += q.x; v.y += q.y; v.z += q.z; v.w += q.w;
    }
    return v;
  };
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  // channels ch .. ch + 3 (on: they exist) over the warp's tokens; put is called by every lane
  auto conv = [&](int ch, bool on, auto &&put) {
    float wt[TAPS][4];
    float4 cur[kDeltaWarpTok], win[TAPS > 1 ? TAPS - 1 : 1];
#pragma unroll
    for (int u = 0; u < kDeltaWarpTok; u++) cur[u] = on && u < nt ? in4(t0 + u, ch) : zero;
#pragma unroll
    for (int j = 0; j < TAPS; j++)
#pragma unroll
      for (int e = 0; e < 4; e++) wt[j][e] = on ? a.cw[(long long)(ch + e) * TAPS + j] : 0.f;
    int prev = -1;
#pragma unroll
    for (int u = 0; u < kDeltaWarpTok; u++) {
      const int t = t0 + u;
      if (u >= nt) break;
      const int s = sp.span[t];
      if (TAPS > 1 && s != prev) {
        prev = s;
        const int back_in_span = t - sp.sp_tok0[s], pos0 = sp.sp_pos0[s];
        const float *tail = a.cstate + (long long)sp.sp_slot[s] * (TAPS - 1) * C + ch;
#pragma unroll
        for (int j = 0; j < TAPS - 1; j++) {
          const int back = TAPS - 1 - j;
          win[j] = !on ? zero : back <= back_in_span ? in4(t - back, ch) : pos0 + back_in_span - back >= 0 ? f4(tail + (long long)((TAPS - 1) - (back - back_in_span)) * C) : zero;
        }
      }
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < TAPS; j++) {
        const float4 v = j + 1 < TAPS ? win[TAPS > 1 && j + 1 < TAPS ? j : 0] : cur[u];
        acc[0] = fmaf(wt[j][0], v.x, acc[0]); acc[1] = fmaf(wt[j][1], v.y, acc[1]); acc[2] = fmaf(wt[j][2], v.z, acc[2]); acc[3] = fmaf(wt[j][3], v.w, acc[3]);
      }
      if (TAPS > 1) {
#pragma unroll
        for (int j = 0; j + 2 < TAPS; j++) win[j] = win[j + 1];
        win[TAPS > 1 ? TAPS - 2 : 0] = cur[u];
      }
      put(t, make_float4(delta_silu(acc[0]), delta_silu(acc[1]), delta_silu(acc[2]), delta_silu(acc[3])));
    }
  };
  int role = blockIdx.y;
  if (role < c.G) {
    const bool on = 4 * l < c.d;
    for (int k = 0; k < 2; k++) {  // query, then key
      const int ch = (k * c.G + role) * c.d + 4 * l;
      const float scale = k ? 1.f : rsqrtf((float)c.d);
      conv(ch, on, [&](int t, float4 v) {
        const float f = rsqrtf(warp_sum(fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)))) + 1e-6f) * scale;
        if (on) *reinterpret_cast<float4 *>(a.buf + (long long)t * a.ld_b + ch) = make_float4(v.x * f, v.y * f, v.z * f, v.w * f);
      });
    }
    return;
  }
  role -= c.G;
  if (role < nvb) {
    const int ch = 2 * c.G * c.d + role * kDeltaTh + 4 * l;
    if (role == 0)
      for (int e = l; e < nt * c.H; e += 32) {
        const int t = t0 + e / c.H, h = e % c.H;
        const float *p = a.proj + (long long)t * a.ld + c.b_off + h;
        float v = p[0];
        for (int k = 1; k < a.n_part; k++) v += p[(long long)k * a.stride];
        a.buf[(long long)t * a.ld_b + C + c.H * c.d + h] = sigmoid_precise(v);
      }
    const bool on = ch < C;
    conv(ch, on, [&](int t, float4 v) { if (on) *reinterpret_cast<float4 *>(a.buf + (long long)t * a.ld_b + ch) = v; });
    return;
  }
  role -= nvb;
  const int n = c.H * c.d, i = role * kDeltaTh + 4 * l;
  if (i >= n) return;
  const float ea = expf(a.vec[i / c.d]);
  float bias[4];
#pragma unroll
  for (int e = 0; e < 4; e++) bias[e] = a.vec[c.H + i + e];
  float4 z[kDeltaWarpTok];
#pragma unroll
  for (int u = 0; u < kDeltaWarpTok; u++) z[u] = u < nt ? f4(a.z + (long long)(t0 + u) * n + i) : zero;
#pragma unroll
  for (int u = 0; u < kDeltaWarpTok; u++) {
    if (u >= nt) break;
    float y[4] = {z[u].x, z[u].y, z[u].z, z[u].w};
#pragma unroll
    for (int e = 0; e < 4; e++) {
      y[e] += bias[e];
      y[e] = expf(-ea * (fmaxf(y[e], 0.f) + log1pf(expf(-fabsf(y[e])))));
    }
    *reinterpret_cast<float4 *>(a.buf + (long long)(t0 + u) * a.ld_b + C + i) = make_float4(y[0], y[1], y[2], y[3]);
  }
}
cudaError_t launch_stack_delta_prep(const StackDelta &c, const StackDeltaPrep &a, bool w_f32, const StackSpans &sp, cudaStream_t st) {
  if (sp.T <= 0) return cudaSuccess;
  if (c.taps < 1 || c.taps > kDeltaMaxTaps) return cudaErrorInvalidValue;
  const int single = sp.T == sp.n_spans ? 1 : 0, tile = single ? 1 : 16;
  const int nvb = (c.H * c.dv + kDeltaTh - 1) / kDeltaTh, ndb = (c.H * c.d + kDeltaTh - 1) / kDeltaTh, ngb = a.z ? 0 : (c.H * c.dv + kDeltaTh - 1) / kDeltaTh;
  auto al = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  if (!single && a.z && c.taps <= 4 && c.d <= 128 && c.d % 4 == 0 && c.dv % 4 == 0 && a.ld % 4 == 0 && a.stride % 4 == 0 && a.ld_b % 4 == 0 && (c.H * c.d) % 4 == 0 && al(a.proj) && al(a.buf) &&
      al(a.z) && al(a.cstate)) {
    const dim3 vgrid((sp.T + kDeltaVecTile - 1) / kDeltaVecTile, c.G + nvb + ndb);
    switch (c.taps) {
      case 1: stack_delta_prep_vec_kernel<1><<<vgrid, kDeltaTh, 0, st>>>(c, a, sp, nvb); break;
      case 2: stack_delta_prep_vec_kernel<2><<<vgrid, kDeltaTh, 0, st>>>(c, a, sp, nvb); break;
      case 3: stack_delta_prep_vec_kernel<3><<<vgrid, kDeltaTh, 0, st>>>(c, a, sp, nvb); break;
      default: stack_delta_prep_vec_kernel<4><<<vgrid, kDeltaTh, 0, st>>>(c, a, sp, nvb);
    }
    DIS_CUDA_TRY(cudaGetLastError());
    return c.taps > 1 ? launch_stack_conv_tail(a.proj, a.ld, a.n_part, a.stride, 0, a.cstate, sp, c.C, c.taps, st) : cudaSuccess;
  }
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
// Four tokens at a time.  With S the state in front of them and G_t = g_1 .. g_t (products of the chunk's decays, per channel),
//   u_t = beta_t (v_t - S^T (G_t k_t) - sum_{s<t} A_ts u_s),   A_ts = sum_i k_t (g_{s+1} .. g_t) k_s,
//   o_t = S^T (G_t q_t) + sum_{s<=t} B_ts u_s,                 B_ts = sum_i q_t (g_{s+1} .. g_t) k_s,
//   S  <- G_4 S + sum_s (g_{s+1} .. g_4) k_s u_s^T
// -- no quotient of decays, so a factor may be zero.  The eight inner products over S do not wait for one another; what has to happen in
// order is six multiplications of numbers per column.  G_t k_t, G_t q_t, the suffix products times k_s, A and B of the next four tokens
// are made while the present ones are worked on (all warps of a CTA share them), and the tokens after those are on their way into
// shared memory.
// The columns of S do not touch each other, so a head is cut into blocks of columns that never exchange anything: a warp owns eight
// columns, each group of eight lanes two of them, and the eight lanes share the rows (RL each, taken in pairs by packed fp32
// operations).  The inner products are added up by a butterfly over the eight lanes that halves the values a lane still carries at
// every step: lanes 0-3 end with a column's products with the k's and solve for u, lanes 4-7 with those with the q's and form o.
// A chunk starts where its span does; tokens beyond the span's end enter as k = q = 0, beta = 0, g = 1.
// State: [slots][H][dv][d], a column's rows next to each other.
// fin.act: the CTA holds whole heads, and each token's o of the head is divided by its root mean square, times norm, times
// sigmoid(gate), and stored in the compute type; else o goes to o [T][H*dv] as it is.
constexpr int kDeltaTok = 4;
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
constexpr int kDeltaVec = 3 * kDeltaTok + 1;  // vectors of a chunk: G_t k_t, G_t q_t, suffix products times k_s, G_4
template <int RL>
constexpr int delta_smem_floats(int nw, int vc) {  // three chunks as they came, vectors and numbers of two, outputs of two
  return 3 * kDeltaTok * (3 * 8 * RL + vc + 4) + 2 * kDeltaVec * 8 * RL + 2 * nw * 16 + nw * 16 + 2 * kDeltaTok * vc;
}
constexpr int kDeltaCols = 2;  // columns of a group of eight lanes
// MW: warps of a CTA at most (fewer leave more registers)
template <int RL, int MW>
__global__ void __launch_bounds__(MW * 32, 1) stack_delta_kernel(StackDelta c, const float *__restrict__ buf, int ld_b, float *state, StackSpans sp,
                                                                 float *__restrict__ o, int ncb, int vec, DeltaFin fin) {
  extern __shared__ __align__(16) float sh[];
  constexpr int DP = 8 * RL, NM = RL / 4, NP = RL / 2, CL = kDeltaCols, CW = 4 * CL, CT = kDeltaTok;
  const int H = c.H, d = c.d, dv = c.dv;
  const int h = blockIdx.x % H, rest = blockIdx.x / H, cb = rest % ncb, s = rest / ncb;  // heads vary fastest: CTAs that run together read whole rows
  const int tok0 = sp.sp_tok0[s], n = sp.sp_len[s], pos0 = sp.sp_pos0[s], slot = sp.sp_slot[s];
  const int NW = blockDim.x >> 5, w = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane & 7, grp = lane >> 3;
  const int NA = min(NW, (d + 31) >> 5);  // warps that prepare chunks
  const int VC = NW * CW, col_cta = cb * VC, nv = min(VC, dv - col_cta);
  const int PT = 3 * DP + VC + 4;  // a token as it comes: q | k | g | v | beta
  float *vecs = sh + 3 * CT * PT;                // [2][kDeltaVec][DP]
  float *part = vecs + 2 * kDeltaVec * DP;       // [2][NW][16]: A and B, a warp's share of the channels
  float *sc = part + 2 * NW * 16 + w * 16;       // [16] A (2,1) (3,1) (3,2) (4,1) (4,2) (4,3), B (t, s) row by row
  float *os = part + 3 * NW * 16;                // [2][CT][VC]
  for (int i = threadIdx.x; i < delta_smem_floats<RL>(NW, VC); i += blockDim.x) sh[i] = 0.f;  // rows beyond d and columns beyond dv stay zero
  const int kvh = h / (H / c.G);
  const int nch = (n + CT - 1) / CT, HV = H * dv;
  // A warp copies whole vectors: q, k, g and v of the chunk's tokens, dealt out from the last warp on (the first ones prepare).  Tokens
  // beyond the span's end: k = q = 0, beta = 0, g = 1.
  const int vcol = 2 * c.G * d + h * dv + col_cta, gcol = c.C + h * d, bcol = c.C + H * d + h;
  const float *rows0 = buf + (long long)tok0 * ld_b;
  auto fetch = [&](int ch) {
    const int left = n - ch * CT;
    const float *rows = rows0 + (long long)(ch * CT) * ld_b;
    float *stage = sh + (ch % 3) * CT * PT;
    for (int job = NW - 1 - w; job < 4 * CT; job += NW) {
      const int tt = job >> 2, which = job & 3;
      float *dst = stage + tt * PT + which * DP;
      const int len = which == 3 ? nv : d;
      if (tt < left) {
        const float *src = rows + tt * ld_b + (which == 0 ? kvh * d : which == 1 ? (c.G + kvh) * d : which == 2 ? gcol : vcol);
        if (vec) for (int e = lane * 4; e < len; e += 128) delta_cp16(dst + e, src + e);
        else for (int e = lane; e < len; e += 32) delta_cp4(dst + e, src + e);
        if (which == 3 && lane == 0) delta_cp4(dst + VC, rows + tt * ld_b + bcol);
      } else {
        for (int e = lane; e < len; e += 32) dst[e] = which == 2 ? 1.f : 0.f;
        if (which == 3 && lane == 0) dst[VC] = 0.f;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // vectors and numbers of chunk ch, a thread per channel
  auto prepare = [&](int ch) {
    if (w >= NA) return;
    const float *raw = sh + (ch % 3) * CT * PT;
    float *vd = vecs + (ch & 1) * kDeltaVec * DP;
    float acc[16];
#pragma unroll
    for (int j = 0; j < 16; j++) acc[j] = 0.f;
    for (int i = threadIdx.x; i < d; i += NA * 32) {
      float q[CT], k[CT], g[CT];
#pragma unroll
      for (int t = 0; t < CT; t++) {
        q[t] = raw[t * PT + i]; k[t] = raw[t * PT + DP + i]; g[t] = raw[t * PT + 2 * DP + i];
      }
      float G = 1.f, suf = 1.f;
#pragma unroll
      for (int t = 0; t < CT; t++) {
        G *= g[t];
        vd[t * DP + i] = G * k[t];
        vd[(CT + t) * DP + i] = G * q[t];
      }
      vd[3 * CT * DP + i] = G;
#pragma unroll
      for (int t = CT - 1; t >= 0; t--) { vd[(2 * CT + t) * DP + i] = suf * k[t]; suf *= g[t]; }
#pragma unroll
      for (int t2 = 0; t2 < CT; t2++) {
        float x = k[t2];
        acc[6 + t2 * (t2 + 1) / 2 + t2] = fmaf(q[t2], x, acc[6 + t2 * (t2 + 1) / 2 + t2]);
#pragma unroll
        for (int t = t2 + 1; t < CT; t++) {
          x *= g[t];
          acc[t * (t - 1) / 2 + t2] = fmaf(k[t], x, acc[t * (t - 1) / 2 + t2]);
          acc[6 + t * (t + 1) / 2 + t2] = fmaf(q[t], x, acc[6 + t * (t + 1) / 2 + t2]);
        }
      }
    }
    const bool c4 = lane & 16, c3 = lane & 8, c2 = lane & 4, c1 = lane & 2;
#pragma unroll
    for (int j = 0; j < 8; j++) acc[j] = (c4 ? acc[j + 8] : acc[j]) + __shfl_xor_sync(0xffffffffu, c4 ? acc[j] : acc[j + 8], 16);
#pragma unroll
    for (int j = 0; j < 4; j++) acc[j] = (c3 ? acc[j + 4] : acc[j]) + __shfl_xor_sync(0xffffffffu, c3 ? acc[j] : acc[j + 4], 8);
#pragma unroll
    for (int j = 0; j < 2; j++) acc[j] = (c2 ? acc[j + 2] : acc[j]) + __shfl_xor_sync(0xffffffffu, c2 ? acc[j] : acc[j + 2], 4);
    acc[0] = (c1 ? acc[1] : acc[0]) + __shfl_xor_sync(0xffffffffu, c1 ? acc[0] : acc[1], 2);
    acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], 1);
    if (!(lane & 1)) part[((ch & 1) * NW + w) * 16 + (lane >> 1)] = acc[0];
  };
  // ---- the state: columns col0 + cc, rows 4 r + 32 m + e
  const int wc = w * CW + grp * CL, col0 = col_cta + wc;
  float *st = state + ((long long)slot * H + h) * dv * d;
  f32x2 S[CL][NP];
#pragma unroll
  for (int cc = 0; cc < CL; cc++) {
    float v[RL];
    const float *p = st + (long long)(col0 + cc) * d;
    const bool on = pos0 > 0 && col0 + cc < dv;
#pragma unroll
    for (int m = 0; m < NM; m++) {
      const int i = r * 4 + 32 * m;
      if (vec) {
        const float4 f = on && i < d ? *reinterpret_cast<const float4 *>(p + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        v[m * 4] = f.x; v[m * 4 + 1] = f.y; v[m * 4 + 2] = f.z; v[m * 4 + 3] = f.w;
      } else {
#pragma unroll
        for (int e = 0; e < 4; e++) v[m * 4 + e] = on && i + e < d ? p[i + e] : 0.f;
      }
    }
#pragma unroll
    for (int q = 0; q < NP; q++) S[cc][q] = pack2(v[2 * q], v[2 * q + 1]);
  }
  auto ld_vec = [&](const float *p, f32x2 (&x)[NP]) {  // this lane's rows of a vector
#pragma unroll
    for (int m = 0; m < NM; m++) {
      const ulonglong2 a = *reinterpret_cast<const ulonglong2 *>(p + r * 4 + 32 * m);
      x[2 * m] = a.x; x[2 * m + 1] = a.y;
    }
  };
  __syncthreads();
  fetch(0);
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  if (nch > 1) fetch(1);
  prepare(0);
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const bool b2 = lane & 4, b1 = lane & 2, b0 = lane & 1;
  const int mycol = (lane >> 1) & 1;  // the column whose sums end in this lane (and its neighbour)
  const bool writes = b2 && !b0 && (fin.act || col0 + mycol < dv);  // this lane forms outputs
  float *op = o + (long long)tok0 * HV + h * dv + col0 + mycol;
  for (int ch = 0; ch < nch; ch++, op += (long long)CT * HV) {
    const int i0 = ch * CT, ct = min(CT, n - i0);
    if (ch + 2 < nch) fetch(ch + 2);
    if (ch + 1 < nch) prepare(ch + 1);
    const float *raw = sh + (ch % 3) * CT * PT, *vd = vecs + (ch & 1) * kDeltaVec * DP;
    if (lane < 16) {
      float v = 0.f;
      for (int k = 0; k < NA; k++) v += part[((ch & 1) * NW + k) * 16 + lane];
      sc[lane] = v;
    }
    float x[CT][CL];
#pragma unroll
    for (int t = 0; t < CT; t++) {
      f32x2 kp[NP], qp[NP];
      ld_vec(vd + t * DP, kp);
      ld_vec(vd + (CT + t) * DP, qp);
#pragma unroll
      for (int cc = 0; cc < CL; cc++) {
        f32x2 a = mul2(S[cc][0], kp[0]), b = mul2(S[cc][0], qp[0]);
#pragma unroll
        for (int q = 1; q < NP; q++) {
          a = fma2(S[cc][q], kp[q], a);
          b = fma2(S[cc][q], qp[q], b);
        }
        float al, ah, bl, bh;
        unpack2(a, al, ah); unpack2(b, bl, bh);
        const float dk = al + ah, dq = bl + bh;
        x[t][cc] = (b2 ? dq : dk) + __shfl_xor_sync(0xffffffffu, b2 ? dk : dq, 4);
      }
    }
#pragma unroll
    for (int t = 0; t < CT; t++) x[t][0] = (b1 ? x[t][1] : x[t][0]) + __shfl_xor_sync(0xffffffffu, b1 ? x[t][0] : x[t][1], 2);
#pragma unroll
    for (int t = 0; t < CT; t++) x[t][0] += __shfl_xor_sync(0xffffffffu, x[t][0], 1);
    __syncwarp();
    float AB[16];
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const float4 f = *reinterpret_cast<const float4 *>(sc + 4 * j);
      AB[4 * j] = f.x; AB[4 * j + 1] = f.y; AB[4 * j + 2] = f.z; AB[4 * j + 3] = f.w;
    }
    float u[CT];  // (lanes 0-3 of a group)
#pragma unroll
    for (int t = 0; t < CT; t++) {
      float y = raw[t * PT + 3 * DP + wc + mycol] - x[t][0];
#pragma unroll
      for (int t2 = 0; t2 < t; t2++) y = fmaf(-AB[t * (t - 1) / 2 + t2], u[t2], y);
      u[t] = raw[t * PT + 3 * DP + VC] * y;
    }
    {
      f32x2 gp[NP];
      ld_vec(vd + 3 * CT * DP, gp);
#pragma unroll
      for (int cc = 0; cc < CL; cc++)
#pragma unroll
        for (int q = 0; q < NP; q++) S[cc][q] = mul2(S[cc][q], gp[q]);
    }
#pragma unroll
    for (int t = 0; t < CT; t++) {
      f32x2 kp[NP];
      ld_vec(vd + (2 * CT + t) * DP, kp);
#pragma unroll
      for (int cc = 0; cc < CL; cc++) {
        const float uc = __shfl_sync(0xffffffffu, u[t], (lane & 24) | (2 * cc));
        const f32x2 u2 = pack2(uc, uc);
#pragma unroll
        for (int q = 0; q < NP; q++) S[cc][q] = fma2(kp[q], u2, S[cc][q]);
      }
    }
#pragma unroll
    for (int t = 0; t < CT; t++) u[t] = __shfl_xor_sync(0xffffffffu, u[t], 4);  // to the lanes that form o
    {
      float *dst = fin.act ? os + (ch & 1) * CT * VC + wc + mycol : op;
      const int step = fin.act ? VC : HV;
#pragma unroll
      for (int t = 0; t < CT; t++) {
        float ov = x[t][0];
#pragma unroll
        for (int t2 = 0; t2 <= t; t2++) ov = fmaf(AB[6 + t * (t + 1) / 2 + t2], u[t2], ov);
        if (writes && t < ct) dst[t * step] = ov;
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (fin.act) {  // a warp finishes a token (columns beyond dv are zero)
      for (int tt = w; tt < ct; tt += NW) {
        const float *ro = os + ((ch & 1) * CT + tt) * VC;
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
      const int i = r * 4 + 32 * m;
      if (vec) {
        if (i < d) *reinterpret_cast<float4 *>(p + i) = make_float4(v[m * 4], v[m * 4 + 1], v[m * 4 + 2], v[m * 4 + 3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; e++)
          if (i + e < d) p[i + e] = v[m * 4 + e];
      }
    }
  }
}

template <int RL, int MW>
static cudaError_t delta_go(const StackDelta &c, const float *buf, long long ld_b, float *state, const StackSpans &sp, float *o, int nw, const float *norm,
                            const float *gate, void *act, long long ld_act, bool f32, uint64_t *launches, cudaStream_t st) {
  const int total = (c.dv + 4 * kDeltaCols - 1) / (4 * kDeltaCols), ncb = (total + nw - 1) / nw, VC = nw * 4 * kDeltaCols;
  const DeltaFin fin{ncb == 1 ? act : nullptr, ld_act, gate, norm, c.eps, f32 ? 1 : 0};
  auto al = [](const void *p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const int vec = c.d % 4 == 0 && c.dv % 4 == 0 && ld_b % 4 == 0 && al(buf) && al(state);
  const size_t shb = (size_t)delta_smem_floats<RL>(nw, VC) * sizeof(float);
  static DeviceOnce once;
  DIS_CUDA_TRY(once.run([&] { return cudaFuncSetAttribute(stack_delta_kernel<RL, MW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024); }));
  stack_delta_kernel<RL, MW><<<(unsigned)((long long)sp.n_spans * c.H * ncb), nw * 32, shb, st>>>(c, buf, (int)ld_b, state, sp, o, ncb, vec, fin);
  DIS_CUDA_TRY(cudaGetLastError());
  *launches += fin.act ? 1 : 2;
  return fin.act ? cudaSuccess : launch_stack_headnorm_silu(o, norm, gate, (long long)c.H * c.dv, act, ld_act, 0, 1.f, f32, sp.T, c.H, c.dv, c.eps, st, true);
}
cudaError_t launch_stack_delta(const StackDelta &c, const float *buf, long long ld_b, float *state, const StackSpans &sp, float *o, int max_len,
                               const float *norm, const float *gate, void *act, long long ld_act, bool f32, uint64_t *launches, cudaStream_t st) {
  if (sp.T <= 0) return cudaSuccess;
  // A head's columns in one CTA (its norm and gate then run inside), but for prompts, where a CTA takes at most eight warps and fewer
  // while halving them still brings idle SMs to work.
  const int total = (c.dv + 4 * kDeltaCols - 1) / (4 * kDeltaCols);
  const bool prompts = max_len > 2 * kDeltaTok;
  int nw = std::min(total, prompts || c.d > 128 ? 8 : 16);
  while (prompts && nw > 4 && (long long)sp.n_spans * c.H * ((total + nw - 1) / nw) * 2 <= 148) nw = (nw + 1) / 2;
#define DIS_DELTA(RL, MW) return delta_go<RL, MW>(c, buf, ld_b, state, sp, o, nw, norm, gate, act, ld_act, f32, launches, st)
  if (nw <= 8) {
    if (c.d <= 32) DIS_DELTA(4, 8);
    if (c.d <= 64) DIS_DELTA(8, 8);
    if (c.d <= 128) DIS_DELTA(16, 8);
    if (c.d <= 256) DIS_DELTA(32, 8);
  } else {
    if (c.d <= 32) DIS_DELTA(4, 16);
    if (c.d <= 64) DIS_DELTA(8, 16);
    if (c.d <= 128) DIS_DELTA(16, 16);
  }
#undef DIS_DELTA
  return cudaErrorInvalidValue;
}

}  // namespace dis

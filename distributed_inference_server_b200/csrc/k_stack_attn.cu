// k_stack_attn.cu -- grouped-query attention over paged keys and values for the layer-list decoders (DIS_MIX_ATTENTION and the
// attention half of DIS_MIX_PARALLEL): the per-token preparation (biases, whole-projection or per-head query/key norm, partial
// rotary with a frequency table, cache write of the rotated keys and of the values -- own projection or the unrotated keys,
// optionally rotated by their position; a layer that reads another layer's cache writes nothing) and the attention itself with
// softmax (optionally with a per-head sink logit in the denominator) or per-head sigmoid weights, under a causal mask that may
// be cut into chunks of positions, over the whole visible history or a slice of it, with an optional per-head sigmoid gate on
// the output.  Scores, weights, norms and angles are fp32 (angles are formed in double) whatever the cache's element type.
#include "stack_dev.cuh"

namespace dis {

// ------------------------------------------------------------------------------------------------ preparation
// One block per token.  proj row: queries at q_off [H][d], keys at k_off [G][d], values at v_off [G][dv] (unless values are
// the keys).  `bias` (or null): one entry per column of the projection, added here when the product left it out.
// kpool == null: the layer reads another layer's cache; only the queries are prepared.
// n_part > 1: the projection comes as split-K slices (slice stride `stride`); the block first sums its token's row of n_cols
// columns (and the bias) into shared memory and works from there.  gate_out (or null): receives columns gate_off .. of the row, H or
// (DIS_ATTN_GATE_FULL) H*dv of them (the logits of the output gates, which the attention kernel reads from memory).
// mix: DIS_ATTN_V_MIX -- the first such layer of a pass leaves its values in mix.save, the later ones blend theirs with them.
template <bool F32>
__global__ void __launch_bounds__(512) stack_attn_prep_kernel(const float *proj, long long ld, int n_part, long long stride, int n_cols,
                                                              int gate_off, float *gate_out, long long ld_gate, int q_off, int k_off, int v_off,
                                                              const float *bias, const float *qn, const float *kn, const double *freq,
                                                              const double *vfreq, StackAttn c, StackSpans sp, float *qf, void *kpool,
                                                              void *vpool, float *vrot, const int *page_table, int max_pages,
                                                              int page_size, StackVMix mix) {
  extern __shared__ __align__(16) float tab[];  // cos [half], sin [half], value cos [dv/2], value sin [dv/2], per-head factors [H + G], summed row
  const int HM = c.H * c.maps, GM = c.G * c.maps;  // heads of queries and keys, each map a head of its own here
  const int srow_off = (c.rot_dims + c.dv + HM + GM + 3) & ~3;  // the summed row starts on a 16-byte boundary
  __shared__ float sh[32];
  const int t = blockIdx.x;
  const float *row = proj + (long long)t * ld;
  if (n_part > 1) {
    float *srow = tab + srow_off;
    if ((((int)(ld & 3)) | (int)(stride & 3) | (n_cols & 3)) == 0) {  // 16-byte loads of every slice, all independent
      for (int i = threadIdx.x * 4; i < n_cols; i += blockDim.x * 4) {
        float4 v = bias ? *reinterpret_cast<const float4 *>(bias + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
        for (int k = 0; k < n_part; k++) {
          const float4 p = *reinterpret_cast<const float4 *>(row + (long long)k * stride + i);
          v.x += p.x; v.y += p.y; v.z += p.z; v.w += p.w;
        }
        *reinterpret_cast<float4 *>(srow + i) = v;
      }
    } else
    for (int i = threadIdx.x; i < n_cols; i += blockDim.x) {
      float v = bias ? bias[i] : 0.f;
      for (int k = 0; k < n_part; k++) v += row[(long long)k * stride + i];
      srow[i] = v;
    }
    row = srow;
    bias = nullptr;
    __syncthreads();
  }
  if (gate_out)
    for (int i = threadIdx.x, n = (c.flags & DIS_ATTN_GATE_FULL) ? c.H * c.dv : c.H; i < n; i += blockDim.x) gate_out[(long long)t * ld_gate + i] = row[gate_off + i];
  const int pos = sp.pos[t], slot = sp.slot[t];
  const int half = c.rot_dims >> 1, vhalf = c.dv >> 1;
  const bool rot_v = (c.flags & DIS_ATTN_ROT_V) != 0, own = kpool != nullptr;
  float *cs = tab, *sn = tab + half, *vcs = sn + half, *vsn = vcs + vhalf, *hr = vsn + vhalf;
  for (int i = threadIdx.x; i < half; i += blockDim.x) angle_sincos(pos, freq[i], &sn[i], &cs[i]);
  if (rot_v)
    for (int i = threadIdx.x; i < vhalf; i += blockDim.x) {
      float s_, c_;
      angle_sincos(pos, vfreq[i], &s_, &c_);
      vcs[i] = c_; vsn[i] = s_;
      vrot[(long long)t * c.dv + i] = c_;
      vrot[(long long)t * c.dv + vhalf + i] = s_;
    }
  const int nq = HM * c.d, nk = GM * c.d;
  const float *qb = bias ? bias + q_off : nullptr, *kb = bias ? bias + k_off : nullptr, *vb = bias ? bias + v_off : nullptr;
  const bool head_norm = (c.flags & DIS_ATTN_QK_NORM_HEAD) != 0;
  float rq = 1.f, rk = 1.f;
  if (c.flags & DIS_ATTN_QK_NORM) {
    float s = 0.f;
    for (int i = threadIdx.x; i < nq; i += blockDim.x) { const float v = row[q_off + i] + (qb ? qb[i] : 0.f); s += v * v; }
    rq = rsqrtf(block_sum(s, sh) / (float)nq + c.eps);
    s = 0.f;
    for (int i = threadIdx.x; i < nk; i += blockDim.x) { const float v = row[k_off + i] + (kb ? kb[i] : 0.f); s += v * v; }
    rk = rsqrtf(block_sum(s, sh) / (float)nk + c.eps);
  } else if (head_norm) {  // one factor per head: a warp per head at a time, query heads then key heads
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
    for (int h = w; h < HM + (own ? GM : 0); h += (int)(blockDim.x >> 5)) {
      const bool isq = h < HM;
      const int off = isq ? q_off + h * c.d : k_off + (h - HM) * c.d;
      const float *b = isq ? (qb ? qb + h * c.d : nullptr) : (kb ? kb + (h - HM) * c.d : nullptr);
      float s = 0.f;
      for (int i = l; i < c.d; i += 32) { const float v = row[off + i] + (b ? b[i] : 0.f); s += v * v; }
      s = warp_sum(s);
      if (l == 0) hr[h] = rsqrtf(s / (float)c.d + c.eps);
    }
  }
  __syncthreads();
  // g: the gain vector (whole projection, or [d] shared by the heads); r / rh: the factor of the projection or of each head
  auto val = [&](int off, const float *b, const float *g, float r, const float *rh, int i) {
    float v = row[off + i] + (b ? b[i] : 0.f);
    if (g) v = head_norm ? v * rh[i / c.d] * g[i % c.d] : v * r * g[i];
    return v;
  };
  auto rotated = [&](int off, const float *b, const float *g, float r, const float *rh, int i) {
    const int e = i % c.d;
    if (e >= c.rot_dims) return val(off, b, g, r, rh, i);
    if (c.flags & DIS_ATTN_ROT_PAIRS) {
      const int p = e >> 1;
      return e & 1 ? val(off, b, g, r, rh, i) * cs[p] + val(off, b, g, r, rh, i - 1) * sn[p] : val(off, b, g, r, rh, i) * cs[p] - val(off, b, g, r, rh, i + 1) * sn[p];
    }
    if (e < half) return val(off, b, g, r, rh, i) * cs[e] - val(off, b, g, r, rh, i + half) * sn[e];
    return val(off, b, g, r, rh, i) * cs[e - half] + val(off, b, g, r, rh, i - half) * sn[e - half];
  };
  const bool normed = (c.flags & (DIS_ATTN_QK_NORM | DIS_ATTN_QK_NORM_HEAD)) != 0;
  const float *qg = normed ? qn : nullptr, *kg = normed ? kn : nullptr;
  for (int i = threadIdx.x; i < nq; i += blockDim.x) qf[(long long)t * nq + i] = rotated(q_off, qb, qg, rq, hr, i);
  if (!own) return;
  const long long prow = (long long)page_table[(long long)slot * max_pages + pos / page_size] * page_size + pos % page_size;
  for (int i = threadIdx.x; i < nk; i += blockDim.x) st_el<F32>(kpool, prow * nk + i, rotated(k_off, kb, kg, rk, hr + HM, i));
  const int nv = c.G * c.dv;
  for (int i = threadIdx.x; i < nv; i += blockDim.x) {
    float v;
    if (c.flags & DIS_ATTN_V_IS_K) v = row[k_off + i] + (kb ? kb[i] : 0.f);  // dv == d: the keys as projected
    else if (!rot_v) v = row[v_off + i] + (vb ? vb[i] : 0.f);
    else {
      const int e = i % c.dv;
      auto vv = [&](int j) { return row[v_off + j] + (vb ? vb[j] : 0.f); };
      v = e < vhalf ? vv(i) * vcs[e] - vv(i + vhalf) * vsn[e] : vv(i) * vcs[e - vhalf] + vv(i - vhalf) * vsn[e - vhalf];
    }
    if (mix.save) mix.save[(long long)t * nv + i] = v;
    if (mix.first) { const float lam = mix.lam[0]; v = (1.f - lam) * v + lam * mix.first[(long long)t * nv + i]; }
    st_el<F32>(vpool, prow * nv + i, v);
  }
}
cudaError_t launch_stack_attn_prep(const float *proj, long long ld, int n_part, long long stride, int n_cols, int gate_off, float *gate_out,
                                   long long ld_gate, int q_off, int k_off, int v_off, const float *bias, const float *qn,
                                   const float *kn, const double *freq, const double *vfreq, const StackAttn &c, const StackSpans &sp,
                                   float *qf, void *kpool, void *vpool, float *vrot, bool f32, const int *page_table, int max_pages,
                                   int page_size, const StackVMix &mix, cudaStream_t st) {
  if (sp.T <= 0) return cudaSuccess;
  if (n_part < 1) n_part = 1;
  const size_t sh = (size_t)(((c.rot_dims + c.dv + (c.H + c.G) * c.maps + 3) & ~3) + (n_part > 1 ? n_cols : 0)) * sizeof(float);
  if (sh > 200 * 1024) return cudaErrorInvalidValue;
  static DeviceOnce once;
  DIS_CUDA_TRY(once.run([&] {
    cudaError_t e = cudaFuncSetAttribute(stack_attn_prep_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    return e != cudaSuccess ? e : cudaFuncSetAttribute(stack_attn_prep_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  }));
  const int th = sp.T <= 148 ? 512 : 128;  // few tokens: a block per token leaves the GPU empty, so the blocks are large
  if (f32) stack_attn_prep_kernel<true><<<sp.T, th, sh, st>>>(proj, ld, n_part, stride, n_cols, gate_off, gate_out, ld_gate, q_off, k_off, v_off, bias, qn, kn, freq, vfreq, c, sp, qf, kpool, vpool, vrot, page_table, max_pages, page_size, mix);
  else stack_attn_prep_kernel<false><<<sp.T, th, sh, st>>>(proj, ld, n_part, stride, n_cols, gate_off, gate_out, ld_gate, q_off, k_off, v_off, bias, qn, kn, freq, vfreq, c, sp, qf, kpool, vpool, vrot, page_table, max_pages, page_size, mix);
  return cudaGetLastError();
}

// ------------------------------------------------------------------------------------------------ attention, fp32 arithmetic
// One CTA per (query block, key/value head, slice of the history).  The block's (token, query head of the group) pairs share
// 32-key tiles staged in shared memory as fp32; one warp per pair at a time: a lane scores one key, then lanes own value
// coordinates.  SIG: weight = sigmoid(score * temp[h] + pb[h]), plain sums.  Otherwise an online softmax (running maximum and
// denominator per pair).  Epilogue (whole history in one CTA) or merge kernel (slices): normalise, rotate the output back by
// the query's position when values were rotated, scale, and store into the mixer's output row.
// A block walks the keys any of its tokens may see: the kept first positions below its window, then everything from the window's
// start k_lo on.  Both runs are numbered through: index v < n_keep is position v, index v >= n_keep is position v + shift, so tiles
// and slices are cut over one gapless range [0, total) and no tile is spent on a short run of kept keys.
struct AttnWalk {
  int n_keep, shift;
  __device__ __forceinline__ AttnWalk(const StackAttn &c, int k_lo) : n_keep(min(c.keep, k_lo)), shift(k_lo - n_keep) {}
  __device__ __forceinline__ int key(int v) const { return v < n_keep ? v : v + shift; }
  __device__ __forceinline__ int total(int last_pos) const { return last_pos + 1 - shift; }
};
constexpr int kAtTile = 32, kAtWarps = 8, kAtMaxSplit = 64;
bool stack_attn_mma_ok(const StackAttn &c, bool f32);
int stack_attn_mma_block_tokens(const StackAttn &c);

struct AttnOut {
  void *out;          // [T][ld] in the compute type; head h at columns off + h * dv
  long long ld;
  int off;
  float scale;        // factor on the output (weight of this mixer inside a parallel layer)
  const float *vrot;  // [T][dv]: cos | sin of the query position's value angles, or null
  const float *gate;  // [T][ldg]: logit of head h's output gate at column h, or null
  long long ldg;
  const float *gate_full;  // [T][ldg]: logit of the gate of head h's coordinate j at column h * dv + j, or null
};
// factor on head h's output at token tok: the mixer's weight times the head's sigmoid gate
__device__ __forceinline__ float attn_out_factor(const AttnOut &o, int tok, int h) {
  return o.gate ? o.scale * sigmoid_precise(o.gate[(long long)tok * o.ldg + h]) : o.scale;
}

template <bool F32>
__device__ __forceinline__ void attn_store(const AttnOut &o, const float *a, float inv, int tok, int h, int dv, int j) {
  float v = a[j] * inv;
  if (o.vrot) {  // rotation by minus the angle: (u, v) -> (u cos + v sin, v cos - u sin)
    const int hf = dv >> 1;
    const float *cs = o.vrot + (long long)tok * dv, *sn = cs + hf;
    v = j < hf ? (a[j] * cs[j] + a[j + hf] * sn[j]) * inv : (a[j] * cs[j - hf] - a[j - hf] * sn[j - hf]) * inv;
  }
  if (o.gate_full) v *= sigmoid_precise(o.gate_full[(long long)tok * o.ldg + (long long)h * dv + j]);
  st_el<F32>(o.out, (long long)tok * o.ld + o.off + (long long)h * dv + j, v * attn_out_factor(o, tok, h));
}

int stack_attn_block_tokens(const StackAttn &c, bool f32) {
  if (stack_attn_mma_ok(c, f32)) return stack_attn_mma_block_tokens(c);
  const int R = c.H / c.G * c.maps;
  int bq = std::max(1, 32 / R);
  while (bq > 1 && ((size_t)kAtTile * (c.d * c.maps + c.dv + 2 + kAtWarps) + (size_t)bq * R * (c.d + c.dv + 2)) * 4 > 200 * 1024) bq >>= 1;
  return bq;
}
static size_t attn_smem(const StackAttn &c, int bq) {
  const int R = c.H / c.G * c.maps;
  return ((size_t)kAtTile * (c.d * c.maps + c.dv + 2 + kAtWarps) + (size_t)bq * R * (c.d + c.dv + 2)) * sizeof(float);
}

template <bool F32, bool SIG>
__global__ void __launch_bounds__(kAtWarps * 32) stack_attn_kernel(const float *qf, const void *kpool, const void *vpool, const float *temp,
                                                                   const float *pb, const float *sink, StackAttn c, StackSpans sp, const int *qb_tok0,
                                                                   const int *qb_len, const int *page_table, int max_pages,
                                                                   int page_size, AttnOut o, int keys_per_split, float *part) {
  extern __shared__ float shm[];
  // with two maps a head counts twice: pair p = ((token * heads of the group) + head) * maps + map, a key row holds both maps
  const int maps = c.maps, d = c.d, dk = d * maps, dv = c.dv, DP = dk + 1, VP = dv + 1, R = c.H / c.G * maps, g = blockIdx.y;
  const int tok0 = qb_tok0[blockIdx.x], nq = qb_len[blockIdx.x];
  const int pairs = nq * R;
  float *kt = shm;                               // [32][DP]
  float *vt = kt + (size_t)kAtTile * DP;         // [32][VP]
  float *qs = vt + (size_t)kAtTile * VP;         // [pairs][d]
  float *acc = qs + (size_t)pairs * d;           // [pairs][dv]
  float *mx = acc + (size_t)pairs * dv;          // [pairs]
  float *dn = mx + pairs;                        // [pairs]
  float *prs = dn + pairs;                       // [warps][32]
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  const int slot = sp.slot[tok0];
  const int last_pos = sp.pos[tok0 + nq - 1];
  for (int i = threadIdx.x; i < pairs * d; i += blockDim.x) {
    const int p = i / d, e = i - p * d;
    qs[i] = qf[((long long)(tok0 + p / R) * c.H * maps + g * R + p % R) * d + e];
  }
  for (int i = threadIdx.x; i < pairs * dv; i += blockDim.x) acc[i] = 0.f;
  const bool with_sink = !SIG && sink && blockIdx.z == 0;
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) { mx[i] = with_sink ? sink[g * R + i % R] : -INFINITY; dn[i] = with_sink ? 1.f : 0.f; }
  const int *pt = page_table + (long long)slot * max_pages;
  const int k_lo = stack_attn_row_lo(c, sp.pos[tok0]);
  const AttnWalk wk(c, k_lo);
  const int k_begin = part ? (int)blockIdx.z * keys_per_split : 0;  // indices of the walk
  const int k_end = part ? min(wk.total(last_pos), k_begin + keys_per_split) : wk.total(last_pos);
  const long long krow = (long long)c.G * dk, vrow = (long long)c.G * dv;
  const bool dist = !SIG && (c.flags & DIS_ATTN_DISTANCE);
  const float inv_cap = c.softcap > 0.f ? 1.f / c.softcap : 0.f;
  for (int k0 = k_begin; k0 < k_end; k0 += kAtTile) {
    const int nk = min(kAtTile, k_end - k0);
    __syncthreads();
    for (int i = threadIdx.x; i < nk * dk; i += blockDim.x) {
      const int kk = i / dk, cc = i - kk * dk, kp = wk.key(k0 + kk);
      const long long prow = (long long)pt[kp / page_size] * page_size + kp % page_size;
      kt[(size_t)kk * DP + cc] = ld_el<F32>(kpool, prow * krow + (long long)g * dk + cc);
    }
    for (int i = threadIdx.x; i < nk * dv; i += blockDim.x) {
      const int kk = i / dv, cc = i - kk * dv, kp = wk.key(k0 + kk);
      const long long prow = (long long)pt[kp / page_size] * page_size + kp % page_size;
      vt[(size_t)kk * VP + cc] = ld_el<F32>(vpool, prow * vrow + (long long)g * dv + cc);
    }
    __syncthreads();
    for (int p = w; p < pairs; p += kAtWarps) {
      const int qpos = sp.pos[tok0 + p / R], h = g * R + p % R;
      const int qlo = stack_attn_row_lo(c, qpos);
      const float *q = qs + (size_t)p * d;
      float sc = -INFINITY;
      const int kp = wk.key(k0 + l);
      if (l < nk && kp <= qpos && (kp >= qlo || kp < c.keep)) {
        const float *kr = kt + (size_t)l * DP + (maps > 1 ? (p & 1) * d : 0);
        float s0 = 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;  // four chains, added at the end: the sum's order is fixed by d alone
        int i = 0;
        for (; i + 3 < d; i += 4) {
          s0 = fmaf(q[i], kr[i], s0); s1 = fmaf(q[i + 1], kr[i + 1], s1);
          s2 = fmaf(q[i + 2], kr[i + 2], s2); s3 = fmaf(q[i + 3], kr[i + 3], s3);
        }
        for (; i < d; i++) s0 = fmaf(q[i], kr[i], s0);
        sc = ((s0 + s1) + (s2 + s3)) * c.scale;
        if (c.softcap > 0.f) sc = c.softcap * tanhf(sc * inv_cap);
        if (dist) sc -= stack_attn_slope(h, c.H) * (float)(qpos - kp);
      }
      float pr, corr = 1.f, psum = 0.f, m_new = 0.f;
      if (SIG) {
        pr = sc == -INFINITY ? 0.f : 1.f / (1.f + expf(-(sc * temp[h] + pb[h])));
      } else {
        const float m_old = mx[p];
        m_new = fmaxf(m_old, warp_max(sc));
        pr = sc == -INFINITY ? 0.f : expf(sc - m_new);
        corr = m_old == -INFINITY ? 0.f : expf(m_old - m_new);  // (m_new is -inf too while a pair has seen nothing: pr = 0 then)
        psum = warp_sum(pr);
      }
      float *a = acc + (size_t)p * dv;
      float *pw = prs + w * kAtTile;  // the tile's weights of this pair: lanes own coordinates below, so every lane reads all
      pw[l] = pr;
      __syncwarp();
      for (int j = l; j < dv; j += 32) {
        float v0 = a[j] * corr, v1 = 0.f, v2 = 0.f, v3 = 0.f;
        int kk = 0;
        for (; kk + 3 < nk; kk += 4) {
          v0 = fmaf(pw[kk], vt[(size_t)kk * VP + j], v0); v1 = fmaf(pw[kk + 1], vt[(size_t)(kk + 1) * VP + j], v1);
          v2 = fmaf(pw[kk + 2], vt[(size_t)(kk + 2) * VP + j], v2); v3 = fmaf(pw[kk + 3], vt[(size_t)(kk + 3) * VP + j], v3);
        }
        for (; kk < nk; kk++) v0 = fmaf(pw[kk], vt[(size_t)kk * VP + j], v0);
        a[j] = (v0 + v1) + (v2 + v3);
      }
      __syncwarp();
      if (!SIG && l == 0) { mx[p] = m_new; dn[p] = dn[p] * corr + psum; }
      __syncwarp();
    }
  }
  __syncthreads();
  if (!part && maps > 1) {  // a warp joins the two maps of a (token, head)
    for (int p = 2 * w; p < pairs; p += 2 * kAtWarps) {
      const float *a1 = acc + (size_t)p * dv, *a2 = a1 + dv;
      const float f1 = 1.f / dn[p], f2 = c.diff_lambda / dn[p + 1];
      float ss = 0.f;
      for (int j = l; j < dv; j += 32) { const float v = a1[j] * f1 - a2[j] * f2; ss = fmaf(v, v, ss); }
      const float k = rsqrtf(warp_sum(ss) / (float)dv + c.eps) * c.diff_out * o.scale;
      const int tok = tok0 + p / R, h = (g * R + p % R) >> 1;
      for (int j = l; j < dv; j += 32) st_el<F32>(o.out, (long long)tok * o.ld + o.off + (long long)h * dv + j, (a1[j] * f1 - a2[j] * f2) * k);
    }
    return;
  }
  if (!part) {
    for (int i = threadIdx.x; i < pairs * dv; i += blockDim.x) {
      const int p = i / dv, j = i - p * dv;
      attn_store<F32>(o, acc + (size_t)p * dv, SIG ? 1.f : 1.f / dn[p], tok0 + p / R, g * R + p % R, dv, j);
    }
    return;
  }
  // slice record per (token, head): dv unnormalised sums, then the slice's maximum and denominator
  for (int i = threadIdx.x; i < pairs * (dv + 2); i += blockDim.x) {
    const int p = i / (dv + 2), j = i - p * (dv + 2);
    float *rec = part + (((long long)blockIdx.z * sp.T + tok0 + p / R) * c.H * maps + g * R + p % R) * (dv + 2);
    rec[j] = j < dv ? acc[(size_t)p * dv + j] : j == dv ? mx[p] : dn[p];
  }
}

// Merge of the slices of one (token, head): softmax: out = sum_s acc_s e^(m_s - M) / sum_s l_s e^(m_s - M); sigmoid: plain sum.
// Slices that lie wholly behind the token (nothing visible) wrote m = -inf, l = 0 and zeros.
template <bool F32, bool SIG>
__global__ void stack_attn_merge_kernel(const float *part, int n_split, int T, int H, int dv, AttnOut o) {
  extern __shared__ float msh[];  // [dv] merged sums, [n_split] factors
  float *a = msh, *ws = msh + dv;
  __shared__ float inv_den;
  const int p = blockIdx.x, tok = p / H, h = p - tok * H;
  const long long stride = (long long)T * H * (dv + 2);
  const float *rec = part + (long long)p * (dv + 2);
  if (!SIG && threadIdx.x < 32) {  // a lane per slice (at most 64): every slice's maximum and denominator are fetched at once
    const int l = threadIdx.x;
    float m[2], d[2], M = -INFINITY, den = 0.f;
#pragma unroll
    for (int u = 0; u < 2; u++) {
      const int s = l + 32 * u;
      m[u] = s < n_split ? rec[s * stride + dv] : -INFINITY;
      d[u] = s < n_split ? rec[s * stride + dv + 1] : 0.f;
      M = fmaxf(M, m[u]);
    }
    M = warp_max(M);
#pragma unroll
    for (int u = 0; u < 2; u++) {
      const int s = l + 32 * u;
      const float w = m[u] == -INFINITY ? 0.f : expf(m[u] - M);
      if (s < n_split) ws[s] = w;
      den = fmaf(d[u], w, den);
    }
    den = warp_sum(den);
    if (l == 0) inv_den = 1.f / den;
  }
  __syncthreads();
  for (int j = threadIdx.x; j < dv; j += blockDim.x) {
    float v = 0.f;
#pragma unroll 8
    for (int s = 0; s < n_split; s++) v = SIG ? v + rec[s * stride + j] : fmaf(rec[s * stride + j], ws[s], v);
    a[j] = v;
  }
  __syncthreads();
  for (int j = threadIdx.x; j < dv; j += blockDim.x) attn_store<F32>(o, a, SIG ? 1.f : inv_den, tok, h, dv, j);
}

// Merge with two maps: one block per (token, head), a warp forms each map's factors; records of the head's maps lie next to each other.
template <bool F32>
__global__ void __launch_bounds__(128) stack_attn_merge_maps_kernel(const float *part, int n_split, int T, int H, int dv, AttnOut o, float lambda,
                                                                    float diff_out, float eps) {
  extern __shared__ float msh[];  // [dv] joined sums, [2][n_split] factors
  float *a = msh, *ws = msh + dv;
  __shared__ float sh[32];
  const int p = blockIdx.x, tok = p / H, h = p - tok * H;
  const long long stride = (long long)T * H * 2 * (dv + 2);
  const float *rec = part + (long long)p * 2 * (dv + 2);
  // the sums of the first slices are requested beside the maxima and denominators
  constexpr int U = 8;
  const int j0 = threadIdx.x;
  float r1[U], r2[U];
#pragma unroll
  for (int s = 0; s < U; s++) {
    const bool on = s < n_split && j0 < dv;
    r1[s] = on ? rec[s * stride + j0] : 0.f;
    r2[s] = on ? rec[s * stride + dv + 2 + j0] : 0.f;
  }
  if (threadIdx.x < 64) {  // factor of a slice: its weight over the map's denominator, the second map's times -lambda
    const int m = threadIdx.x >> 5, l = threadIdx.x & 31;
    const float *rm = rec + m * (dv + 2);
    float mx[2], d[2], M = -INFINITY, den = 0.f;
#pragma unroll
    for (int u = 0; u < 2; u++) {
      const int s = l + 32 * u;
      mx[u] = s < n_split ? rm[s * stride + dv] : -INFINITY;
      d[u] = s < n_split ? rm[s * stride + dv + 1] : 0.f;
      M = fmaxf(M, mx[u]);
    }
    M = warp_max(M);
#pragma unroll
    for (int u = 0; u < 2; u++) {
      mx[u] = mx[u] == -INFINITY ? 0.f : expf(mx[u] - M);
      den = fmaf(d[u], mx[u], den);
    }
    const float f = (m ? -lambda : 1.f) / warp_sum(den);
#pragma unroll
    for (int u = 0; u < 2; u++)
      if (l + 32 * u < n_split) ws[m * n_split + l + 32 * u] = mx[u] * f;
  }
  __syncthreads();
  float ss = 0.f;
  for (int j = j0; j < dv; j += blockDim.x) {
    float v1 = 0.f, v2 = 0.f;
    if (j == j0) {
#pragma unroll
      for (int s = 0; s < U; s++)
        if (s < n_split) { v1 = fmaf(r1[s], ws[s], v1); v2 = fmaf(r2[s], ws[n_split + s], v2); }
    }
#pragma unroll 8
    for (int s = j == j0 ? U : 0; s < n_split; s++) {
      v1 = fmaf(rec[s * stride + j], ws[s], v1);
      v2 = fmaf(rec[s * stride + dv + 2 + j], ws[n_split + s], v2);
    }
    a[j] = v1 + v2;
    ss = fmaf(a[j], a[j], ss);
  }
  const float k = rsqrtf(block_sum(ss, sh) / (float)dv + eps) * diff_out * o.scale;
  for (int j = j0; j < dv; j += blockDim.x) st_el<F32>(o.out, (long long)tok * o.ld + o.off + (long long)h * dv + j, a[j] * k);
}

// ------------------------------------------------------------------------------------------------ attention on mma.sync
// The bf16 compute type with dim a multiple of 8, vdim a multiple of 16, both at most 128, and at most 64 query heads per
// key/value head.  A CTA of four warps owns up to 64 rows -- the (token, query head of the group) pairs of its query block,
// 16 per warp -- and walks the history in tiles of 64 keys: K and V rows of the pages are copied with cp.async into two
// shared-memory stages (the next tile is in flight while this one is used), S = Q K^T and O += P V run on m16n8k16 with fp32
// accumulators, the weights in between are fp32 (online softmax per row, or the sigmoid form) and are rounded to bf16 only as
// the operand of P V.  Slices and the epilogue are those of the kernel above.
constexpr int kMmKeys = 64, kMmWarps = 4, kMmRows = 16 * kMmWarps;
constexpr float kLog2e = 1.4426950408889634f, kLn2 = 0.6931471805599453f;

__device__ __forceinline__ void mma_bf16_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src, int src_bytes) {  // src_bytes 0: zeros
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(src_bytes));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {  // round to nearest even, one instruction
  uint32_t r;
  asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r) : "f"(hi), "f"(lo));
  return r;
}
__device__ __forceinline__ float ex2_(float x) {  // 2^x, flushing results below the normal range to zero; 2^(-inf) = 0
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

// Scores of one 64-key tile -> sigmoid weights, or scaled scores and the rows' running maxima (softmax).  MASKED: the tile
// reaches past a row's position or the slice's end, or starts before a row's chunk, so every element is checked; interior tiles
// skip the checks.
// cap2 > 0 (softmax only): the scaled score s passes cap tanh(s / cap) first; scale2 is then the plain scale over the cap, and
// tanh x = 1 - 2 / (1 + e^(2x)) is formed with one ex2 and one reciprocal (absolute error of the order of 1e-7, times the cap).
// k0: index of the tile's first key in the walk `wk`; keep: positions below it are always visible.  DIST: the score is lowered by
// slope2[e] per position of distance (slope in units of log 2).
template <bool SIG, bool MASKED, bool DIST>
__device__ __forceinline__ void attn_tile_weights(float (&sacc)[kMmKeys / 8][4], float (&mnew)[2], int k0, int qd, const int (&r_pos)[2],
                                                  const int (&r_lo)[2], int k_end, const AttnWalk &wk, int keep, const float (&tmp_h)[2],
                                                  const float (&pb_h)[2], const float (&slope2)[2], float scale2, float cap2) {
#pragma unroll
  for (int j = 0; j < kMmKeys / 8; j++)
#pragma unroll
    for (int q4 = 0; q4 < 4; q4++) {
      const int e = q4 >> 1;
      bool vis = true;
      const int v = k0 + j * 8 + qd * 2 + (q4 & 1);
      int kp = v + wk.shift;  // (a tile that needs no mask holds no kept keys from below the window)
      if (MASKED) { kp = wk.key(v); vis = kp <= r_pos[e] && v < k_end && (kp >= r_lo[e] || kp < keep); }
      float sv = sacc[j][q4];
      if (SIG) {
        float rc;
        asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(rc) : "f"(1.f + ex2_(-fmaf(sv, tmp_h[e], pb_h[e]))));
        sv = vis ? rc : 0.f;
      } else {
        sv *= scale2;
        if (cap2 > 0.f) {
          float rc;
          asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(rc) : "f"(1.f + ex2_(sv * (2.f * kLog2e))));
          sv = cap2 * fmaf(-2.f, rc, 1.f);
        }
        if (DIST) sv = fmaf(-slope2[e], (float)(r_pos[e] - kp), sv);
        sv = vis ? sv : -INFINITY;
        mnew[e] = fmaxf(mnew[e], sv);
      }
      sacc[j][q4] = sv;
    }
}

bool stack_attn_mma_ok(const StackAttn &c, bool f32) {
  return !f32 && c.d % 8 == 0 && c.dv % 16 == 0 && c.d <= 128 && c.dv <= 128 && c.H / c.G <= kMmRows;
}
int stack_attn_mma_block_tokens(const StackAttn &c) { return std::max(1, kMmRows / (c.H / c.G)); }

// Where the keys and values of a head lie: row r of position p is lin[slot] + p (gathered rows) or, lin null, the row of p's page.  A
// key is its first dk coordinates at k + r * k_ld + head * k_hs, then (k2, shared by the heads) the rest at k2 + r * k2_ld.
struct AttnKV {
  const uint16_t *k, *k2, *v;
  long long k_ld, k2_ld, v_ld;
  int k_hs, dk, v_hs;
  const int *lin;
};
// DQ, DV: compiled sizes of a query / key (of one map) and of a value (the layer's are at most these).
// DIFF: two maps per head (StackAttn::maps).  Twice the warps: warp w and warp w + kMmWarps own the same rows, the first with map 1, the
// second with map 2; a key row in shared memory holds both maps, the value rows are shared.  At the end the second map's outputs go
// through shared memory to the warps of the first, which join, norm and store.  Slice records: maps of a head next to each other.
template <int DQ, int DV, bool SIG, bool DIST, bool DIFF = false>
__global__ void __launch_bounds__(kMmWarps * 32 * (DIFF ? 2 : 1), DIFF ? (DQ > 64 ? 1 : 2) : DQ > 128 ? 2 : 3) stack_attn_mma_kernel(const float *__restrict__ qf, long long ldq, AttnKV kv, const float *temp,
                                                                       const float *pb, const float *sink, StackAttn c, StackSpans sp, const int *qb_tok0,
                                                                       const int *qb_len, const int *page_table, int max_pages,
                                                                       int page_size, AttnOut o, int keys_per_split, float *part) {
  constexpr int KP = DQ * (DIFF ? 2 : 1) + 8, VP = DV + 8;  // elements per shared row: 16-byte rows land in distinct bank groups
  extern __shared__ __align__(16) uint16_t smem[];
  uint16_t *Ks = smem;                               // [2][64][KP]
  uint16_t *Vs = smem + 2 * kMmKeys * KP;            // [2][64][VP]
  const int d = c.d, dv = c.dv, R = c.H / c.G, kvh = blockIdx.y;
  // the blocks of a span come in ascending position, and the later ones walk a longer history: taking the grid backwards starts
  // the long ones first, so the last CTAs to start are short
  const int qb = gridDim.x - 1 - blockIdx.x;
  const int tok0 = qb_tok0[qb], nq = qb_len[qb], rows = nq * R;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, qd = lane & 3;
  const int slot = sp.slot[tok0], pos_first = sp.pos[tok0], last_pos = pos_first + nq - 1;
  const int *pt = page_table + (long long)slot * max_pages;
  // chunked or windowed mask: the first token's bound is where the block's history starts (later rows may start later still)
  const int k_lo = stack_attn_row_lo(c, pos_first);
  const AttnWalk wk(c, k_lo);
  const int k_begin = part ? (int)blockIdx.z * keys_per_split : 0;  // indices of the walk
  const int k_end = part ? min(wk.total(last_pos), k_begin + keys_per_split) : wk.total(last_pos);
  constexpr int NTR = DIFF ? 4 : 2;  // threads that copy a key row
  const int krow_d = DIFF ? 2 * d : d;
  const int nk16 = (d + 15) >> 4, nv8 = dv >> 3, dc = krow_d >> 3, vc = dv >> 3;  // k-steps of Q K^T, n-tiles of P V, 16-byte chunks per row
  // columns d .. 16 nk16 of the K stages are read by the last k-step: zero them once (cp.async never touches them)
  if (d & 15)
    for (int i = threadIdx.x; i < 2 * kMmKeys * 8; i += blockDim.x) Ks[(i >> 3) * KP + krow_d + (i & 7)] = 0;
  const int rwarp = DIFF ? warp & (kMmWarps - 1) : warp, map = DIFF ? warp / kMmWarps : 0;
  // ---- this thread's rows: r0 = 16 rwarp + gid and r0 + 8
  int r_tok[2], r_head[2], r_pos[2], r_lo[2];
  bool r_ok[2];
  uint32_t qa[DQ / 16][4];
#pragma unroll
  for (int e = 0; e < 2; e++) {
    const int r = rwarp * 16 + gid + e * 8;
    r_ok[e] = r < rows;
    r_tok[e] = tok0 + (r_ok[e] ? r / R : 0);
    r_head[e] = kvh * R + (r_ok[e] ? r % R : 0);
    r_pos[e] = r_ok[e] ? pos_first + r / R : -1;
    r_lo[e] = r_ok[e] ? stack_attn_row_lo(c, r_pos[e]) : 0;
  }
#pragma unroll
  for (int ks = 0; ks < DQ / 16; ks++) {
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const float *qr = qf + (long long)r_tok[e] * ldq + (long long)(DIFF ? 2 * r_head[e] + map : r_head[e]) * d;
#pragma unroll
      for (int hf = 0; hf < 2; hf++) {
        const int col = ks * 16 + hf * 8 + qd * 2;
        float x0 = 0.f, x1 = 0.f;
        if (r_ok[e] && ks < nk16) {
          if (col < d) x0 = qr[col];
          if (col + 1 < d) x1 = qr[col + 1];
        }
        qa[ks][hf * 2 + e] = pack_bf16(x0, x1);
      }
    }
  }
  float oacc[DV / 8][4];
#pragma unroll
  for (int j = 0; j < DV / 8; j++) { oacc[j][0] = oacc[j][1] = oacc[j][2] = oacc[j][3] = 0.f; }
  float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};
  if (!SIG && sink && blockIdx.z == 0) {  // the sink term of the denominator enters as the initial state of the first slice (one lane of the four holds its 1)
#pragma unroll
    for (int e = 0; e < 2; e++) { mrow[e] = sink[r_head[e]] * kLog2e; lrow[e] = qd == 0 ? 1.f : 0.f; }
  }
  float tmp_h[2] = {1.f, 1.f}, pb_h[2] = {0.f, 0.f};
  if (SIG) {
#pragma unroll
    for (int e = 0; e < 2; e++) { tmp_h[e] = temp[r_head[e]] * c.scale * kLog2e; pb_h[e] = pb[r_head[e]] * kLog2e; }
  }
  float slope2[2] = {0.f, 0.f};
  if (DIST) {
#pragma unroll
    for (int e = 0; e < 2; e++) slope2[e] = stack_attn_slope(r_head[e], c.H) * kLog2e;
  }
  // with a soft cap the scores are first brought to units of the cap (scale / cap), and the capped score to units of log 2
  const float cap2 = !SIG && c.softcap > 0.f ? c.softcap * kLog2e : 0.f;
  const float scale2 = cap2 > 0.f ? c.scale / c.softcap : c.scale * kLog2e;
  const bool warp_live = rwarp * 16 < rows;
  const int warp_last_pos = pos_first + min(rows - 1, rwarp * 16 + 15) / R;
  const int warp_first_pos = pos_first + (rwarp * 16) / R;
  const int warp_lo = stack_attn_row_lo(c, warp_first_pos);        // first key any row of the warp sees
  const int warp_lo_max = stack_attn_row_lo(c, warp_last_pos);     // first key every row of the warp sees
  const uint16_t *kh = kv.k + (long long)kvh * kv.k_hs, *vh = kv.v + (long long)kvh * kv.v_hs;
  const int dk8 = kv.dk >> 3;
  const long long lin0 = kv.lin ? kv.lin[slot] : 0;
  const uint32_t ks_base = (uint32_t)__cvta_generic_to_shared(Ks), vs_base = (uint32_t)__cvta_generic_to_shared(Vs);
  // NTR threads per key row: one page-table read per thread and tile, then the row's 16-byte chunks alternate between them
  const int ld_row = threadIdx.x / NTR, ld_part = threadIdx.x % NTR;
  const int pshift = 31 - __clz(page_size);  // page_size is a power of two
  // the page of this thread's row is read one tile ahead of the copy that needs it
  auto page_of = [&](int k0) { const int v = k0 + ld_row; return v < k_end && !kv.lin ? pt[wk.key(v) >> pshift] : 0; };
  int page_next = page_of(k_begin);
  auto load_tile = [&](int k0, int stage) {
    const int kp = wk.key(k0 + ld_row);
    const bool ok = k0 + ld_row < k_end;
    const long long prow = !ok ? 0 : kv.lin ? lin0 + kp : (long long)page_next * page_size + (kp & (page_size - 1));
    page_next = page_of(k0 + kMmKeys);
    const uint16_t *ksrc = kh + prow * kv.k_ld, *vsrc = vh + prow * kv.v_ld;
    const uint32_t kdst = ks_base + (uint32_t)(((stage * kMmKeys + ld_row) * KP) * 2), vdst = vs_base + (uint32_t)(((stage * kMmKeys + ld_row) * VP) * 2);
#pragma unroll 4
    for (int ch = ld_part; ch < dk8; ch += NTR) cp_async16(kdst + ch * 16, ksrc + ch * 8, ok ? 16 : 0);
    if (dk8 < dc) {  // the shared part of the key
      const uint16_t *k2 = kv.k2 + prow * kv.k2_ld;
      for (int ch = dk8 + ld_part; ch < dc; ch += NTR) cp_async16(kdst + ch * 16, k2 + (ch - dk8) * 8, ok ? 16 : 0);
    }
#pragma unroll 4
    for (int ch = ld_part; ch < vc; ch += NTR) cp_async16(vdst + ch * 16, vsrc + ch * 8, ok ? 16 : 0);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int n_tiles = k_end > k_begin ? (k_end - k_begin + kMmKeys - 1) / kMmKeys : 0;
  if (n_tiles > 0) load_tile(k_begin, 0);
  for (int it = 0; it < n_tiles; it++) {
    const int k0 = k_begin + it * kMmKeys, stage = it & 1;
    if (it + 1 < n_tiles) {
      load_tile(k0 + kMmKeys, stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int key_a = wk.key(k0), key_z = wk.key(k0 + kMmKeys - 1);  // positions of the tile's first and last key
    if (warp_live && key_a <= warp_last_pos && (key_z >= warp_lo || key_a < c.keep)) {
      // S = Q K^T: k-steps outside, key tiles inside, so that consecutive products go to different accumulators; one ldmatrix
      // brings the fragments of two key tiles (lane l: matrix l / 8 = (tile, column half), row l % 8)
      const uint32_t kt = ks_base + (uint32_t)((stage * kMmKeys * KP + (DIFF ? map * d : 0)) * 2);
      float sacc[kMmKeys / 8][4];
#pragma unroll
      for (int j = 0; j < kMmKeys / 8; j++) { sacc[j][0] = sacc[j][1] = sacc[j][2] = sacc[j][3] = 0.f; }
#pragma unroll
      for (int ks = 0; ks < DQ / 16; ks++) {
        if (ks < nk16) {
#pragma unroll
          for (int j = 0; j < kMmKeys / 8; j += 2) {
            uint32_t b0, b1, b2, b3;
            ldsm_x4(kt + (uint32_t)((((j + (lane >> 4)) * 8 + (lane & 7)) * KP + ks * 16 + ((lane >> 3) & 1) * 8) * 2), b0, b1, b2, b3);
            mma_bf16_16816(sacc[j], qa[ks], b0, b1);
            mma_bf16_16816(sacc[j + 1], qa[ks], b2, b3);
          }
        }
      }
      // ---- weights, fp32.  Scores are carried in units of log 2 (the factor 1 / ln 2 is folded into the scale), so every
      // exponential is one ex2.  Only a tile that reaches past a row's position or the slice's end needs the mask.
      const bool masked = key_z > warp_first_pos || k0 + kMmKeys > k_end || key_a < warp_lo_max;
      float mnew[2] = {mrow[0], mrow[1]};
      if (masked) attn_tile_weights<SIG, true, DIST>(sacc, mnew, k0, qd, r_pos, r_lo, k_end, wk, c.keep, tmp_h, pb_h, slope2, scale2, cap2);
      else attn_tile_weights<SIG, false, DIST>(sacc, mnew, k0, qd, r_pos, r_lo, k_end, wk, c.keep, tmp_h, pb_h, slope2, scale2, cap2);
      if (!SIG) {
        float corr[2];
#pragma unroll
        for (int e = 0; e < 2; e++) {
          mnew[e] = fmaxf(mnew[e], __shfl_xor_sync(0xffffffffu, mnew[e], 1));
          mnew[e] = fmaxf(mnew[e], __shfl_xor_sync(0xffffffffu, mnew[e], 2));
          corr[e] = mrow[e] == -INFINITY ? 0.f : ex2_(mrow[e] - mnew[e]);
          mrow[e] = mnew[e];
          lrow[e] *= corr[e];
        }
        const float msub[2] = {mnew[0] == -INFINITY ? 0.f : mnew[0], mnew[1] == -INFINITY ? 0.f : mnew[1]};  // a row with nothing visible yet
#pragma unroll
        for (int j = 0; j < kMmKeys / 8; j++)
#pragma unroll
          for (int q4 = 0; q4 < 4; q4++) {
            const int e = q4 >> 1;
            const float pv = ex2_(sacc[j][q4] - msub[e]);  // 2^(-inf) = 0 for the masked
            sacc[j][q4] = pv;
            lrow[e] += pv;
          }
#pragma unroll
        for (int j = 0; j < DV / 8; j++) { oacc[j][0] *= corr[0]; oacc[j][1] *= corr[0]; oacc[j][2] *= corr[1]; oacc[j][3] *= corr[1]; }
      }
      // ---- O += P V
      const uint32_t vt = vs_base + (uint32_t)(stage * kMmKeys * VP * 2);
#pragma unroll
      for (int kk = 0; kk < kMmKeys / 16; kk++) {
        uint32_t pa[4];
        pa[0] = pack_bf16(sacc[2 * kk][0], sacc[2 * kk][1]);
        pa[1] = pack_bf16(sacc[2 * kk][2], sacc[2 * kk][3]);
        pa[2] = pack_bf16(sacc[2 * kk + 1][0], sacc[2 * kk + 1][1]);
        pa[3] = pack_bf16(sacc[2 * kk + 1][2], sacc[2 * kk + 1][3]);
#pragma unroll
        for (int j = 0; j < DV / 8; j += 2) {
          if (j < nv8) {
            // lanes 0-15: keys 16 kk + lane of columns 8 j; lanes 16-31: the same keys of columns 8 (j + 1)
            uint32_t b0, b1, b2, b3;
            ldsm_x4_trans(vt + (uint32_t)(((kk * 16 + (lane & 15)) * VP + (j + (lane >> 4)) * 8) * 2), b0, b1, b2, b3);
            mma_bf16_16816(oacc[j], pa, b0, b1);
            mma_bf16_16816(oacc[j + 1], pa, b2, b3);
          }
        }
      }
    }
    __syncthreads();
  }
  if (!SIG) {
#pragma unroll
    for (int e = 0; e < 2; e++) {
      lrow[e] += __shfl_xor_sync(0xffffffffu, lrow[e], 1);
      lrow[e] += __shfl_xor_sync(0xffffffffu, lrow[e], 2);
    }
  }
  if (DIFF && !part) {  // (the last tile's barrier has passed: the stages are free)
    float *o2 = reinterpret_cast<float *>(smem);  // [64 rows][DV + 4]: the second map's normalised outputs
    if (map == 1 && warp_live) {
#pragma unroll
      for (int e = 0; e < 2; e++) {
        const float inv = 1.f / lrow[e];
        float *orow = o2 + (size_t)(rwarp * 16 + gid + e * 8) * (DV + 4) + qd * 2;
#pragma unroll
        for (int j = 0; j < DV / 8; j++)
          if (j < nv8) *reinterpret_cast<float2 *>(orow + j * 8) = make_float2(oacc[j][e * 2] * inv, oacc[j][e * 2 + 1] * inv);
      }
    }
    __syncthreads();
    if (map == 1) return;
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const float inv = 1.f / lrow[e];
      const float *orow = o2 + (size_t)(rwarp * 16 + gid + e * 8) * (DV + 4) + qd * 2;
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < DV / 8; j++)
        if (j < nv8) {
          const float2 v = *reinterpret_cast<const float2 *>(orow + j * 8);
          oacc[j][e * 2] = fmaf(-c.diff_lambda, v.x, oacc[j][e * 2] * inv);
          oacc[j][e * 2 + 1] = fmaf(-c.diff_lambda, v.y, oacc[j][e * 2 + 1] * inv);
          ss = fmaf(oacc[j][e * 2], oacc[j][e * 2], fmaf(oacc[j][e * 2 + 1], oacc[j][e * 2 + 1], ss));
        }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      const float k = rsqrtf(ss / (float)dv + c.eps) * c.diff_out * o.scale;
      if (!r_ok[e]) continue;
      uint16_t *out = reinterpret_cast<uint16_t *>(o.out) + (long long)r_tok[e] * o.ld + o.off + (long long)r_head[e] * dv + qd * 2;
#pragma unroll
      for (int j = 0; j < DV / 8; j++)
        if (j < nv8) *reinterpret_cast<uint32_t *>(out + j * 8) = pack_bf16(oacc[j][e * 2] * k, oacc[j][e * 2 + 1] * k);
    }
    return;
  }
  // ---- results: thread holds, for row e, columns 8 j + 2 qd + {0, 1} of every n-tile j
  if (!part && o.vrot) {
    // rotation back by the query's position pairs column m with m + dv/2: the warp's 16 x dv tile goes through shared memory
    // (every key tile has been consumed; a warp reads only the rows it wrote)
    float *ot = reinterpret_cast<float *>(smem) + (size_t)warp * 16 * (dv + 1);
#pragma unroll
    for (int e = 0; e < 2; e++) {
#pragma unroll
      for (int j = 0; j < DV / 8; j++)
        if (j < nv8) { ot[(gid + e * 8) * (dv + 1) + j * 8 + qd * 2] = oacc[j][e * 2]; ot[(gid + e * 8) * (dv + 1) + j * 8 + qd * 2 + 1] = oacc[j][e * 2 + 1]; }
      if (qd == 0) ot[(gid + e * 8) * (dv + 1) + dv] = attn_out_factor(o, r_tok[e], r_head[e]) * (SIG ? 1.f : 1.f / lrow[e]);
    }
    __syncwarp();
    const int hf = dv >> 1;
    for (int i = lane; i < 16 * hf; i += 32) {
      const int rr = i / hf, m = i - rr * hf, r = warp * 16 + rr;
      if (r >= rows) continue;
      const int tok = tok0 + r / R, head = kvh * R + r % R;
      const float *cs = o.vrot + (long long)tok * dv, *sn = cs + hf;
      const float u = ot[rr * (dv + 1) + m], w = ot[rr * (dv + 1) + m + hf], inv = ot[rr * (dv + 1) + dv];
      uint16_t *orow = reinterpret_cast<uint16_t *>(o.out) + (long long)tok * o.ld + o.off + (long long)head * dv;
      float a0 = (u * cs[m] + w * sn[m]) * inv, a1 = (w * cs[m] - u * sn[m]) * inv;
      if (o.gate_full) {
        const float *gr = o.gate_full + (long long)tok * o.ldg + (long long)head * dv;
        a0 *= sigmoid_precise(gr[m]); a1 *= sigmoid_precise(gr[m + hf]);
      }
      orow[m] = float_to_bf16_bits(a0);
      orow[m + hf] = float_to_bf16_bits(a1);
    }
    return;
  }
#pragma unroll
  for (int e = 0; e < 2; e++) {
    if (!r_ok[e]) continue;
    if (part) {
      float *rec = part + (((long long)blockIdx.z * sp.T + r_tok[e]) * c.H + r_head[e]) * (dv + 2) * (DIFF ? 2 : 1) + (DIFF ? map * (dv + 2) : 0);
#pragma unroll
      for (int j = 0; j < DV / 8; j++)
        if (j < nv8) { rec[j * 8 + qd * 2] = oacc[j][e * 2]; rec[j * 8 + qd * 2 + 1] = oacc[j][e * 2 + 1]; }
      if (qd == 0) { rec[dv] = SIG ? 0.f : mrow[e] * kLn2; rec[dv + 1] = lrow[e]; }  // the maximum back in natural units
      continue;
    }
    const float inv = attn_out_factor(o, r_tok[e], r_head[e]) * (SIG ? 1.f : 1.f / lrow[e]);
    uint16_t *orow = reinterpret_cast<uint16_t *>(o.out) + (long long)r_tok[e] * o.ld + o.off + (long long)r_head[e] * dv;
    const float *gr = o.gate_full ? o.gate_full + (long long)r_tok[e] * o.ldg + (long long)r_head[e] * dv + qd * 2 : nullptr;
#pragma unroll
    for (int j = 0; j < DV / 8; j++)
      if (j < nv8) {
        float a0 = oacc[j][e * 2] * inv, a1 = oacc[j][e * 2 + 1] * inv;
        if (gr) { a0 *= sigmoid_precise(gr[j * 8]); a1 *= sigmoid_precise(gr[j * 8 + 1]); }
        *reinterpret_cast<uint32_t *>(orow + j * 8 + qd * 2) = pack_bf16(a0, a1);
      }
  }
}

static cudaError_t attn_mma_go(const float *qf, long long ldq, const AttnKV &kv, const float *temp, const float *pb, const float *sink,
                               const StackAttn &c, const StackSpans &sp, const int *qb_tok0, const int *qb_len, dim3 grid, const int *page_table,
                               int max_pages, int page_size, const AttnOut &o, int keys_per_split, float *part, cudaStream_t st) {
  static DeviceOnce once;
  DIS_CUDA_TRY(once.run([&] {
    cudaError_t e = cudaSuccess;
    auto allow = [&](auto kern) { if (e == cudaSuccess) e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024); };
    allow(stack_attn_mma_kernel<64, 64, true, false>);
    allow(stack_attn_mma_kernel<64, 64, false, false>);
    allow(stack_attn_mma_kernel<64, 64, false, true>);
    allow(stack_attn_mma_kernel<128, 128, true, false>);
    allow(stack_attn_mma_kernel<128, 128, false, false>);
    allow(stack_attn_mma_kernel<128, 128, false, true>);
    allow(stack_attn_mma_kernel<192, 128, false, false>);
    allow(stack_attn_mma_kernel<64, 64, false, false, true>);
    allow(stack_attn_mma_kernel<64, 128, false, false, true>);
    allow(stack_attn_mma_kernel<128, 128, false, false, true>);
    return e;
  }));
  const bool sig = (c.flags & DIS_ATTN_SIGMOID) != 0, dist = (c.flags & DIS_ATTN_DISTANCE) != 0;
  const bool small = c.d <= 64 && c.dv <= 64;
  const int dq = small ? 64 : c.d <= 128 ? 128 : 192, dvp = small ? 64 : 128;
  if (c.maps > 1) {
    if (sig || dist || c.d > 128 || c.dv > 128) return cudaErrorInvalidValue;
    const int dqm = c.d <= 64 ? 64 : 128, dvm = small ? 64 : 128;
    const size_t shd = std::max((size_t)2 * kMmKeys * (2 * dqm + dvm + 16) * sizeof(uint16_t), (size_t)kMmRows * (dvm + 4) * sizeof(float));
#define DIS_ATTN_DIFF_MMA(Q, V) \
  stack_attn_mma_kernel<Q, V, false, false, true><<<grid, kMmWarps * 64, shd, st>>>(qf, ldq, kv, temp, pb, nullptr, c, sp, qb_tok0, qb_len, page_table, max_pages, page_size, o, keys_per_split, part)
    if (dqm == 64 && dvm == 64) DIS_ATTN_DIFF_MMA(64, 64);
    else if (dqm == 64) DIS_ATTN_DIFF_MMA(64, 128);
    else DIS_ATTN_DIFF_MMA(128, 128);
#undef DIS_ATTN_DIFF_MMA
    return cudaGetLastError();
  }
  if (c.d > dq || c.dv > dvp || (dq == 192 && (sig || dist))) return cudaErrorInvalidValue;
  const size_t shm = (size_t)2 * kMmKeys * (dq + dvp + 16) * sizeof(uint16_t);
#define DIS_ATTN_MMA(Q, V, S, B) \
  stack_attn_mma_kernel<Q, V, S, B><<<grid, kMmWarps * 32, shm, st>>>(qf, ldq, kv, temp, pb, sink, c, sp, qb_tok0, qb_len, page_table, max_pages, page_size, o, keys_per_split, part)
  if (dq == 192) DIS_ATTN_MMA(192, 128, false, false);
  else if (small && sig) DIS_ATTN_MMA(64, 64, true, false);
  else if (small && dist) DIS_ATTN_MMA(64, 64, false, true);
  else if (small) DIS_ATTN_MMA(64, 64, false, false);
  else if (sig) DIS_ATTN_MMA(128, 128, true, false);
  else if (dist) DIS_ATTN_MMA(128, 128, false, true);
  else DIS_ATTN_MMA(128, 128, false, false);
#undef DIS_ATTN_MMA
  return cudaGetLastError();
}

// Latent attention of prompt portions on the same kernel: every head has keys and values of its own, made from the gathered latents
// (kv [rows][H*(d + dv)]: all heads' unrotated key parts, then all heads' values), and the rotated key part krot [rows][dr] is shared.
// Position p of the sequence in slot s is row lin[s] + p.
bool stack_latent_flash_ok(const StackLatent &c, bool f32) {
  return !f32 && c.r % 8 == 0 && c.d % 8 == 0 && c.dr % 8 == 0 && c.dv % 16 == 0 && c.d + c.dr <= 192 && c.dv <= 128;
}
int stack_latent_flash_tokens() { return kMmRows; }
cudaError_t launch_stack_latent_flash(const float *q, long long ldq, const uint16_t *kv, const uint16_t *krot, const int *lin, const float *sink,
                                      const StackLatent &c, const StackSpans &sp, const int *qb_tok0, const int *qb_len, int n_qb, void *out,
                                      long long ld_out, const float *gate, long long ld_gate, cudaStream_t st) {
  if (n_qb <= 0) return cudaSuccess;
  const StackAttn a{c.H, c.H, c.d + c.dr, c.dv, 0, 0u, c.scale, c.eps, 0, c.window};
  const long long ld = (long long)c.H * (c.d + c.dv);
  const AttnKV src{kv, krot, kv + (long long)c.H * c.d, ld, (long long)c.dr, ld, c.d, c.d, c.dv, lin};
  const AttnOut o{out, ld_out, 0, 1.f, nullptr, nullptr, ld_gate, gate};
  return attn_mma_go(q, ldq, src, nullptr, nullptr, sink, a, sp, qb_tok0, qb_len, dim3(n_qb, c.H, 1), nullptr, 0, 1, o, 0, nullptr, st);
}

cudaError_t launch_stack_attn(const float *qf, const void *kpool, const void *vpool, bool f32, const float *temp, const float *pb,
                              const float *sink, const StackAttn &c, const StackSpans &sp, const int *qb_tok0, const int *qb_len, int n_qb,
                              int bq, const int *page_table, int max_pages, int page_size, void *out, long long ld_out, int out_off,
                              float out_scale, const float *vrot, const float *gate, long long ld_gate, int n_split,
                              int keys_per_split, float *part, cudaStream_t st) {
  if (n_qb <= 0) return cudaSuccess;
  if (!(c.flags & (DIS_ATTN_SINK | DIS_ATTN_SINK_UNIT))) sink = nullptr;  // the unit sink is a vector of zero logits
  const float *gate_full = (c.flags & DIS_ATTN_GATE_FULL) ? gate : nullptr;
  if (!(c.flags & DIS_ATTN_GATE)) gate = nullptr;
  if (n_split <= 1 || !part) { n_split = 1; part = nullptr; }
  if (n_split > kAtMaxSplit) return cudaErrorInvalidValue;
  const bool sig = (c.flags & DIS_ATTN_SIGMOID) != 0;
  const size_t sh = attn_smem(c, bq);
  if (sh > 220 * 1024) return cudaErrorInvalidValue;
  static DeviceOnce once;
  DIS_CUDA_TRY(once.run([&] {
    cudaError_t e = cudaFuncSetAttribute(stack_attn_kernel<true, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(stack_attn_kernel<true, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(stack_attn_kernel<false, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
    return e != cudaSuccess ? e : cudaFuncSetAttribute(stack_attn_kernel<false, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  }));
  const AttnOut o{out, ld_out, out_off, out_scale, (c.flags & DIS_ATTN_ROT_V) ? vrot : nullptr, gate, ld_gate, gate_full};
  const dim3 grid(n_qb, c.G, n_split);
  static int use_mma = -1;
  if (use_mma < 0) { const char *e = getenv("DIS_STACK_ATTN_MMA"); use_mma = (e && atoi(e) == 0) ? 0 : 1; }
  // the output's 4-byte stores want even columns; bq is the block size the pass was planned with
  if (use_mma && stack_attn_mma_ok(c, f32) && bq <= stack_attn_mma_block_tokens(c) && ld_out % 2 == 0 && out_off % 2 == 0) {
    const uint16_t *kp = reinterpret_cast<const uint16_t *>(kpool), *vp = reinterpret_cast<const uint16_t *>(vpool);
    const int dk = c.d * c.maps;
    const AttnKV kv{kp, nullptr, vp, (long long)c.G * dk, 0, (long long)c.G * c.dv, dk, dk, c.dv, nullptr};
    DIS_CUDA_TRY(attn_mma_go(qf, (long long)c.H * dk, kv, temp, pb, sink, c, sp, qb_tok0, qb_len, grid, page_table, max_pages, page_size, o, keys_per_split, part, st));
    if (part) {
      const size_t msh = (size_t)(c.dv + n_split) * sizeof(float);
      if (c.maps > 1)
        stack_attn_merge_maps_kernel<false><<<sp.T * c.H, 128, msh + n_split * sizeof(float), st>>>(part, n_split, sp.T, c.H, c.dv, o, c.diff_lambda, c.diff_out, c.eps);
      else if (sig) stack_attn_merge_kernel<false, true><<<sp.T * c.H, 128, msh, st>>>(part, n_split, sp.T, c.H, c.dv, o);
      else stack_attn_merge_kernel<false, false><<<sp.T * c.H, 128, msh, st>>>(part, n_split, sp.T, c.H, c.dv, o);
    }
    return cudaGetLastError();
  }
  const int th = kAtWarps * 32;
#define DIS_ATTN_LAUNCH(F, S) \
  stack_attn_kernel<F, S><<<grid, th, sh, st>>>(qf, kpool, vpool, temp, pb, sink, c, sp, qb_tok0, qb_len, page_table, max_pages, page_size, o, keys_per_split, part)
  if (f32 && sig) DIS_ATTN_LAUNCH(true, true);
  else if (f32) DIS_ATTN_LAUNCH(true, false);
  else if (sig) DIS_ATTN_LAUNCH(false, true);
  else DIS_ATTN_LAUNCH(false, false);
#undef DIS_ATTN_LAUNCH
  if (part) {
    const size_t msh = (size_t)(c.dv + n_split) * sizeof(float);
    const int rows = sp.T * c.H;
    if (c.maps > 1) {
      if (f32) stack_attn_merge_maps_kernel<true><<<rows, 128, msh + n_split * sizeof(float), st>>>(part, n_split, sp.T, c.H, c.dv, o, c.diff_lambda, c.diff_out, c.eps);
      else stack_attn_merge_maps_kernel<false><<<rows, 128, msh + n_split * sizeof(float), st>>>(part, n_split, sp.T, c.H, c.dv, o, c.diff_lambda, c.diff_out, c.eps);
    } else if (f32 && sig) stack_attn_merge_kernel<true, true><<<rows, 64, msh, st>>>(part, n_split, sp.T, c.H, c.dv, o);
    else if (f32) stack_attn_merge_kernel<true, false><<<rows, 64, msh, st>>>(part, n_split, sp.T, c.H, c.dv, o);
    else if (sig) stack_attn_merge_kernel<false, true><<<rows, 64, msh, st>>>(part, n_split, sp.T, c.H, c.dv, o);
    else stack_attn_merge_kernel<false, false><<<rows, 64, msh, st>>>(part, n_split, sp.T, c.H, c.dv, o);
  }
  return cudaGetLastError();
}

}  // namespace dis

// Further mechanisms of the decoder-LM handle (dlm.cu), first used by the Megolorn design: differential softmax attention on the
// query's own chunk of positions (two query / key maps per head over the same values), its query / key / value preparation with
// a bias, a norm per head and map and rotary positions, gated feed-forward units that share the preparation's launch, and a
// router with a choice correction, groups and identity experts.  The attention kernels take one map as well (with a learned bias by
// distance and a gate per element: the Korirax design).
//   T = activation / weight / cache type (bf16, or float in the all-fp32 mode).  Norms, positions and angles, scores and
//   attention weights, routers, lambda and the residual stream are fp32 in both modes.
#pragma once

#include <algorithm>

#include "dlm_mixers2.cuh"

namespace b200 {
namespace dlm {

// cos and sin of pos * freq[i] (evaluated in double), times amp: rot[token] = [half] cosines, [half] sines.  One launch per step
// serves every layer with this rotation.
__global__ void __launch_bounds__(64) rotary_table_kernel(const int* __restrict__ tok_pos, const double* __restrict__ freq, int half, float amp,
                                                          float* __restrict__ rot) {
  rotary_fill(rot + (long long)blockIdx.x * 2 * half, half, tok_pos[blockIdx.x], freq, amp);
}

// what stands between a feed-forward's two products: a bounded or a silu gate times the value, or the value's erf GELU (no gate)
enum { GLU_CLAMPED = 0, GLU_SILU = 1, UNIT_GELU_ERF = 2 };
__device__ __forceinline__ float gelu_erff(float z) { return 0.5f * z * (1.f + erff(z * 0.7071067811865476f)); }
__device__ __forceinline__ float gated_unit(float g, float u, int kind, float limit) {
  return kind == GLU_CLAMPED ? clamped_gluf(g, u, limit) : kind == GLU_SILU ? g * sigmoidf(g) * u : gelu_erff(u);
}

// act[c] = gated_unit(row[off_g + c], row[off_u + c]) on the columns [c0, c0 + GLU_SLICE) of one token, 256 threads
constexpr int GLU_SLICE = 2048;
struct UnitParams {
  int off_g, off_u, F, kind; float limit;      // off_g = off_u where there is no gate
  void* act; long long lda;                    // T
};
template <typename T>
__device__ __forceinline__ void unit_slice(const UnitParams& p, const T* __restrict__ row, long long ld, long long t, int c0) {
  const int c1 = min(p.F, c0 + GLU_SLICE);
  T* act = static_cast<T*>(p.act) + t * p.lda;
  if (sizeof(T) == 2 && ((p.F | p.off_g | p.off_u) & 7) == 0 && ((ld | p.lda) & 7) == 0 && ((uintptr_t)p.act & 15) == 0) {
    for (int c = c0 + threadIdx.x * 8; c < c1; c += 256 * 8) {
      const uint4 gv = *reinterpret_cast<const uint4*>(row + p.off_g + c), uv = *reinterpret_cast<const uint4*>(row + p.off_u + c);
      const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gv);
      const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&uv);
      uint4 ov;
      unsigned* o = reinterpret_cast<unsigned*>(&ov);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float2 g = __bfloat1622float2(g2[k]), u = __bfloat1622float2(u2[k]);
        o[k] = pack_bf16(gated_unit(g.x, u.x, p.kind, p.limit), gated_unit(g.y, u.y, p.kind, p.limit));
      }
      *reinterpret_cast<uint4*>(act + c) = ov;
    }
  } else {
    for (int c = c0 + threadIdx.x; c < c1; c += 256) act[c] = from_f<T>(gated_unit(to_f(row[p.off_g + c]), to_f(row[p.off_u + c]), p.kind, p.limit));
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Preparation of the attention and of the gated feed-forward beside it, on the concatenated projection proj T [tokens][ld].
// grid (tokens, head_rows + slices).  The first head_rows rows of the grid, one warp per (head, map): x + bias, / rms over dim * w (when w is given), rotated,
// queries times qscale (and 1 + temp_coef ln(floor((pos + 1) / temp_every) + 1) where temp_every > 0) -> qout TQ [tokens][Hm * dim], keys -> cache row (off_k < 0: the layer has no keys and values); values +
// bias -> cache row.  The rows after them: the feed-forward's unit on GLU_SLICE columns each.
// ---------------------------------------------------------------------------------------------------------------------------
struct HeadPrepParams {
  const void* proj; long long ld;       // T
  int off_q, off_k, off_v, Hm, Gm, Nv;  // Hm = query heads * maps, Gm = key heads * maps
  int dim, half, adjacent;
  const float* rot;                     // [tokens][2 * half]
  const float* bias;                    // [Hm * dim | Gm * dim | Nv] or null
  const float *wq, *wk;                 // [dim] or null
  float eps, qscale;
  void* qout;                           // TQ
  void *kcache, *vcache; int cap;       // T
  const int *tok_slot, *tok_pos;
  UnitParams unit;
  int head_rows;
  float temp_coef = 0.f, temp_every = 0.f;
};

template <typename T, typename TQ>
__global__ void __launch_bounds__(256) head_prep_kernel(HeadPrepParams p) {
  extern __shared__ float prep_buf[];   // [8 warps][dim]
  const long long t = blockIdx.x;
  const T* row = static_cast<const T*>(p.proj) + t * p.ld;
  if ((int)blockIdx.y >= p.head_rows) {
    unit_slice<T>(p.unit, row, p.ld, t, ((int)blockIdx.y - p.head_rows) * GLU_SLICE);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, dim = p.dim;
  const float* rot = p.rot + t * 2 * p.half;
  const long long crow = (long long)p.tok_slot[t] * p.cap + p.tok_pos[t];
  float* buf = prep_buf + warp * dim;
  const int n = p.Hm + (p.off_k >= 0 ? p.Gm : 0);
  for (int hm = blockIdx.y * 8 + warp; hm < n; hm += p.head_rows * 8) {
    const bool key = hm >= p.Hm;
    const int i = key ? hm - p.Hm : hm;
    const T* src = row + (key ? p.off_k : p.off_q) + i * dim;
    const float* b = p.bias ? p.bias + hm * dim : nullptr;
    const float* w = key ? p.wk : p.wq;
    float ss = 0.f;
    for (int e = lane; e < dim; e += 32) {
      const float x = to_f(src[e]) + (b ? b[e] : 0.f);
      buf[e] = x;
      ss = fmaf(x, x, ss);
    }
    if (w) {
      const float r = 1.f / sqrtf(warp_sum(ss) / (float)dim + p.eps);
      for (int e = lane; e < dim; e += 32) buf[e] *= r * w[e];
    }
    __syncwarp();
    if (key) {
      T* kc = static_cast<T*>(p.kcache) + crow * p.Gm * dim + i * dim;
      for (int e = lane; e < dim; e += 32) kc[e] = from_f<T>(rotary_at<float>(buf, e, p.half, p.adjacent, rot));
    } else {
      const float qs = p.qscale * (p.temp_every > 0.f ? 1.f + p.temp_coef * logf(floorf((float)(p.tok_pos[t] + 1) / p.temp_every) + 1.f) : 1.f);
      TQ* qo = static_cast<TQ*>(p.qout) + t * p.Hm * dim + i * dim;
      for (int e = lane; e < dim; e += 32) qo[e] = from_f<TQ>(rotary_at<float>(buf, e, p.half, p.adjacent, rot) * qs);
    }
    __syncwarp();
  }
  if (p.off_k >= 0 && blockIdx.y == 0) {
    T* vc = static_cast<T*>(p.vcache) + crow * p.Nv;
    const float* b = p.bias ? p.bias + (p.Hm + p.Gm) * dim : nullptr;
    for (int e = threadIdx.x; e < p.Nv; e += 256) vc[e] = from_f<T>(to_f(row[p.off_v + e]) + (b ? b[e] : 0.f));
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Attention with NM query / key maps per head over the same values, NM = 2: differential attention, NM = 1: one softmax.  Rows are (token, query head of ONE key/value head g) pairs, head fastest: row = token * rep + r,
// query head g * rep + r.  A tile is up to MR such rows of one request (tokens may be cut anywhere); every (tile, g) is a CTA of
// its own.  Per map m = 0, 1:  s_m[j] = q_m . k_m[j]  (q carries the scale),  lo <= j <= pos,  lo = start of pos's chunk (or 0);
// a_m = softmax(s_m) . V;   NM = 2: o = a_0 - lambda a_1;   out = o / sqrt(mean(o^2) + eps) * out_scale * sigmoid(gate).
// NM = 1: s[j] += bias[head][min(pos - j, far)] (when bias is given: the table over distances, constant from `far` on);
// out = a_0 * sigmoid(egate) element by element (when given).
// Cache rows: keys T [slots][cap][G][NM][dim], values T [slots][cap][G][vdim].
// nsplit > 1 (grid.y): the key tiles are dealt over the splits, which leave per row [O_m .. | m_m l_m ..] (sums of
// exp(s - m) v, running maximum, sum) for map_attn_merge_kernel.
// ---------------------------------------------------------------------------------------------------------------------------
struct MapAttnParams {
  const void* q; long long ldq;         // bf16 (tensor-core kernel) or fp32 [tokens][H][NM][dim]
  const void *kcache, *vcache;
  const int *tile_row0, *tile_rows, *tile_slot, *tok_pos;
  const float* gate; long long ldg;     // [tokens][ldg] gate pre-activations, null: none
  void* out; long long ldo;             // T [tokens][ldo], head h at h * vdim
  float* part;                          // [tile][g][split][MR][NM * (vdim + 2)]
  int cap, H, G, dim, vdim, chunk, nsplit, n_tiles, MR, KT;
  float lambda, out_scale, eps;
  const float* bias = nullptr; int far = 0;      // [H][far + 1]
  int bias_smem = 0;                             // tensor-core kernel: offset of a shared copy of the rows in use (0: read from global memory)
  const void* egate = nullptr; long long lde = 0;      // T [tokens][lde], head h at h * vdim
};

__device__ __forceinline__ int chunk_start(int pos, int chunk) { return chunk > 0 ? pos / chunk * chunk : 0; }

// one row per warp: value(c) is the maps' combined result; every lane calls
template <typename T, int NM, typename F>
__device__ __forceinline__ void map_row_out(const MapAttnParams& p, int g, long long row, int lane, F value) {
  const int rep = p.H / p.G;
  const long long tok = row / rep;
  const int head = g * rep + (int)(row - tok * rep);
  T* out = static_cast<T*>(p.out) + tok * p.ldo + (long long)head * p.vdim;
  if constexpr (NM == 1) {
    const T* eg = p.egate ? static_cast<const T*>(p.egate) + tok * p.lde + (long long)head * p.vdim : nullptr;
    for (int c = lane; c < p.vdim; c += 32) out[c] = from_f<T>(value(c) * (eg ? sigmoidf(to_f(eg[c])) : 1.f));
    return;
  }
  float ss = 0.f;
  for (int c = lane; c < p.vdim; c += 32) { const float o = value(c); ss = fmaf(o, o, ss); }
  float f = p.out_scale / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
  if (p.gate) f *= sigmoidf(p.gate[tok * p.ldg + head]);
  for (int c = lane; c < p.vdim; c += 32) out[c] = from_f<T>(value(c) * f);
}

// CUDA cores, any sizes, fp32 arithmetic on T caches.  Shared memory: queries, accumulators, scores, staged keys and values.
inline size_t map_attn_smem(int nm, int dim, int vdim, int MR, int KT) {
  return 4 * ((size_t)MR * nm * dim + (size_t)MR * nm * vdim + (size_t)MR * nm * (KT + 1) + (size_t)3 * MR * nm + (size_t)KT * (nm * dim + 1) + (size_t)KT * vdim);
}

template <typename T, int NM>
__global__ void __launch_bounds__(256) map_attn_kernel(MapAttnParams p) {
  extern __shared__ float da_smem[];
  const int dim = p.dim, vdim = p.vdim, MR = p.MR, KT = p.KT, rep = p.H / p.G, D2 = NM * dim, KS = D2 + 1, SS = KT + 1;
  float* qs = da_smem;                                 // [MR][NM][dim]
  float* oacc = qs + MR * D2;                          // [MR][NM][vdim]
  float* sc = oacc + MR * NM * vdim;                    // [MR][NM][SS]
  float* rm = sc + MR * NM * SS;                        // [MR][NM] running maximum, sum, correction
  float* rl = rm + MR * NM;
  float* rc = rl + MR * NM;
  float* ks = rc + MR * NM;                             // [KT][KS]
  float* vs = ks + KT * KS;                            // [KT][vdim]
  const int tile = p.n_tiles - 1 - (int)blockIdx.x / p.G, g = blockIdx.x % p.G, split = blockIdx.y;
  const long long row0 = p.tile_row0[tile];
  const int rows = p.tile_rows[tile], warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* kc = static_cast<const T*>(p.kcache) + (long long)p.tile_slot[tile] * p.cap * p.G * D2 + g * D2;
  const T* vc = static_cast<const T*>(p.vcache) + (long long)p.tile_slot[tile] * p.cap * p.G * vdim + g * vdim;
  const int kmin = chunk_start(p.tok_pos[row0 / rep], p.chunk), kmax = p.tok_pos[(row0 + rows - 1) / rep];
  const int n_kt = (kmax - kmin) / KT + 1, per = (n_kt + p.nsplit - 1) / p.nsplit;
  const int kt0 = split * per, kt1 = min(n_kt, kt0 + per);
  for (int i = threadIdx.x; i < MR * D2; i += 256) {
    const int r = i / D2, e = i - r * D2;
    float v = 0.f;
    if (r < rows) {
      const long long tok = (row0 + r) / rep;
      v = static_cast<const float*>(p.q)[tok * p.ldq + (long long)(g * rep + (int)(row0 + r - tok * rep)) * D2 + e];
    }
    qs[i] = v;
  }
  for (int i = threadIdx.x; i < MR * NM * vdim; i += 256) oacc[i] = 0.f;
  for (int i = threadIdx.x; i < MR * NM; i += 256) { rm[i] = -INFINITY; rl[i] = 0.f; }
  for (int kt = kt0; kt < kt1; ++kt) {
    const int kb = kmin + kt * KT, nk = min(KT, kmax + 1 - kb);
    __syncthreads();
    for (int i = threadIdx.x; i < nk * D2; i += 256) { const int j = i / D2, e = i - j * D2; ks[j * KS + e] = to_f(kc[(long long)(kb + j) * p.G * D2 + e]); }
    for (int i = threadIdx.x; i < nk * vdim; i += 256) { const int j = i / vdim, e = i - j * vdim; vs[i] = to_f(vc[(long long)(kb + j) * p.G * vdim + e]); }
    __syncthreads();
    for (int i = threadIdx.x; i < rows * NM * KT; i += 256) {      // scores, keys fastest
      const int rmi = i / KT, j = i - rmi * KT, r = rmi / NM, m = rmi % NM;
      const int pos = p.tok_pos[(row0 + r) / rep];
      float s = -INFINITY;
      if (j < nk && kb + j <= pos && kb + j >= chunk_start(pos, p.chunk)) {
        const float *qv = qs + r * D2 + m * dim, *kv = ks + j * KS + m * dim;
        s = 0.f;
        for (int d = 0; d < dim; ++d) s = fmaf(qv[d], kv[d], s);
        if (NM == 1 && p.bias) s += p.bias[(long long)(g * rep + (int)((row0 + r) % rep)) * (p.far + 1) + min(pos - (kb + j), p.far)];
      }
      sc[rmi * SS + j] = s;
    }
    __syncthreads();
    for (int rmi = warp; rmi < rows * NM; rmi += 8) {              // online softmax, one warp per (row, map)
      float mx = -INFINITY;
      for (int j = lane; j < KT; j += 32) mx = fmaxf(mx, sc[rmi * SS + j]);
      const float mo = rm[rmi], mn = fmaxf(mo, warp_max(mx));
      float sum = 0.f;
      for (int j = lane; j < KT; j += 32) {
        const float s = sc[rmi * SS + j], w = s > -INFINITY ? expf(s - mn) : 0.f;
        sc[rmi * SS + j] = w;
        sum += w;
      }
      sum = warp_sum(sum);
      __syncwarp();
      if (lane == 0) {
        const float corr = mo > -INFINITY ? expf(mo - mn) : 0.f;
        rc[rmi] = corr; rl[rmi] = rl[rmi] * corr + sum; rm[rmi] = mn;
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < rows * NM * vdim; i += 256) {
      const int rmi = i / vdim, c = i - rmi * vdim;
      const float* w = sc + rmi * SS;
      float acc = oacc[i] * rc[rmi];
      for (int j = 0; j < nk; ++j) acc = fmaf(w[j], vs[j * vdim + c], acc);
      oacc[i] = acc;
    }
  }
  __syncthreads();
  if (p.nsplit == 1) {
    for (int r = warp; r < rows; r += 8) {
      const float* a0 = oacc + r * NM * vdim;
      const float i0 = 1.f / rl[NM * r];
      if constexpr (NM == 1) {
        map_row_out<T, 1>(p, g, row0 + r, lane, [&](int c) { return a0[c] * i0; });
      } else {
        const float* a1 = a0 + vdim;
        const float i1 = p.lambda / rl[2 * r + 1];
        map_row_out<T, 2>(p, g, row0 + r, lane, [&](int c) { return a0[c] * i0 - a1[c] * i1; });
      }
    }
  } else {
    constexpr int E = 2 * NM;           // a row's maxima and sums behind its values
    const int PS = NM * vdim + E;
    float* dst = p.part + (((long long)tile * p.G + g) * p.nsplit + split) * MR * PS;
    for (int i = threadIdx.x; i < rows * NM * vdim; i += 256) { const int r = i / (NM * vdim); dst[(long long)r * PS + (i - r * NM * vdim)] = oacc[i]; }
    for (int i = threadIdx.x; i < rows * NM; i += 256) {
      float* d = dst + (long long)(i / NM) * PS + NM * vdim + 2 * (i % NM);
      d[0] = rm[i]; d[1] = rl[i];
    }
  }
}

// merges the key splits, one warp per row; grid (tiles * G, rows / 4)
template <typename T, int NM>
__global__ void __launch_bounds__(128) map_attn_merge_kernel(MapAttnParams p) {
  const int tile = blockIdx.x / p.G, g = blockIdx.x % p.G, r = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= p.tile_rows[tile]) return;
  const int vdim = p.vdim, PS = NM * (vdim + 2);
  const float* base = p.part + (((long long)tile * p.G + g) * p.nsplit * p.MR + r) * PS;
  const long long ss = (long long)p.MR * PS;
  float f[NM][2];      // lane s: weights of split s and s + 32 for every map
  for (int m = 0; m < NM; ++m) {
    const float ma = lane < p.nsplit ? base[lane * ss + NM * vdim + 2 * m] : -INFINITY, la = lane < p.nsplit ? base[lane * ss + NM * vdim + 2 * m + 1] : 0.f;
    const float mb = lane + 32 < p.nsplit ? base[(lane + 32) * ss + NM * vdim + 2 * m] : -INFINITY, lb = lane + 32 < p.nsplit ? base[(lane + 32) * ss + NM * vdim + 2 * m + 1] : 0.f;
    const float M = warp_max(fmaxf(ma, mb));
    const float ea = ma > -INFINITY ? expf(ma - M) : 0.f, eb = mb > -INFINITY ? expf(mb - M) : 0.f;
    const float inv = (m ? -p.lambda : 1.f) / warp_sum(ea * la + eb * lb);
    f[m][0] = ea * inv; f[m][1] = eb * inv;
  }
  // the row's combined values, a lane's columns c = lane + 32 i, summed over the splits in order; vdim <= 32 * 32 (checked on the host)
  float o[32];
#pragma unroll
  for (int i = 0; i < 32; ++i) o[i] = 0.f;
  for (int s = 0; s < p.nsplit; ++s) {
    const float w0 = __shfl_sync(0xffffffffu, s < 32 ? f[0][0] : f[0][1], s & 31), w1 = NM == 1 ? 0.f : __shfl_sync(0xffffffffu, s < 32 ? f[NM - 1][0] : f[NM - 1][1], s & 31);
    const float* src = base + s * ss;
#pragma unroll
    for (int i = 0; i < 32; ++i)
      if (lane + 32 * i < vdim) o[i] += NM == 1 ? w0 * src[lane + 32 * i] : w0 * src[lane + 32 * i] + w1 * src[vdim + lane + 32 * i];
  }
  const int rep = p.H / p.G;
  const long long row = p.tile_row0[tile] + r, tok = row / rep;
  const int head = g * rep + (int)(row - tok * rep);
  if constexpr (NM == 1) {
    T* out = static_cast<T*>(p.out) + tok * p.ldo + (long long)head * vdim;
    const T* eg = p.egate ? static_cast<const T*>(p.egate) + tok * p.lde + (long long)head * vdim : nullptr;
#pragma unroll
    for (int i = 0; i < 32; ++i)
      if (lane + 32 * i < vdim) out[lane + 32 * i] = from_f<T>(o[i] * (eg ? sigmoidf(to_f(eg[lane + 32 * i])) : 1.f));
    return;
  }
  float q = 0.f;
#pragma unroll
  for (int i = 0; i < 32; ++i) q = fmaf(o[i], o[i], q);
  float k = p.out_scale / sqrtf(warp_sum(q) / (float)vdim + p.eps);
  if (p.gate) k *= sigmoidf(p.gate[tok * p.ldg + head]);
  T* out = static_cast<T*>(p.out) + tok * p.ldo + (long long)head * vdim;
#pragma unroll
  for (int i = 0; i < 32; ++i)
    if (lane + 32 * i < vdim) out[lane + 32 * i] = from_f<T>(o[i] * k);
}

// ---------------------------------------------------------------------------------------------------------------------------
// The same attention on the tensor cores for bf16 caches (dim and vdim multiples of 16, vdim <= VT * 16 <= 128), 64-key tiles
// copied asynchronously into two buffers.  SK = false (prompts): 64 rows, a warp owns 16 of them and walks all keys; both maps'
// scores and weights stay in registers (the scores' accumulator layout is the weights' operand layout) and one fragment of the
// values feeds both maps' sums.  SK = true (single tokens): 16 rows, the warps share them and take 16 keys of a tile each, with
// running maxima of their own that meet in shared memory at the end.
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int DA_KT = 64;
__device__ __forceinline__ float exp2_approx(float x) {      // the hardware exponential (2 ulp; results below the normal range become 0)
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
inline size_t map_attn_mma_smem(int nm, int dim, int VT, bool sk) {
  const size_t qs = nm * dim + 8, vs = VT * 16 + 8, mr = sk ? 16 : 64;
  const size_t tiles = 2 * (mr * qs + 2 * DA_KT * qs + 2 * DA_KT * vs);
  const size_t meet = sk ? 4 * ((size_t)4 * nm * 16 * (VT * 16 + 4) + 4 * nm * 16 * 2) : 0;
  return std::max(tiles, meet);
}

template <int NM, int VT, bool SK>
__global__ void __launch_bounds__(128, 2) map_attn_mma_kernel(MapAttnParams p) {
  constexpr int MR = SK ? 16 : 64, KT = DA_KT, NP = SK ? 1 : 4, VS = VT * 16 + 8;
  constexpr float L2E = 1.4426950408889634f;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int dim = p.dim, vdim = p.vdim, rep = p.H / p.G, D2 = NM * dim, QS = D2 + 8;
  bf16* Qs = reinterpret_cast<bf16*>(smem_raw);                   // [MR][QS]
  bf16* Ks = Qs + MR * QS;                                        // [2][KT][QS]
  bf16* Vs = Ks + 2 * KT * QS;                                    // [2][KT][VS]
  // the last tiles of a prompt see the most keys: they are started first
  const int tile = p.n_tiles - 1 - (int)blockIdx.x / p.G, g = blockIdx.x % p.G, split = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g8 = lane >> 2, t4 = lane & 3, mi = lane >> 3;
  const int row0 = p.tile_row0[tile], rows = p.tile_rows[tile];
  const long long NK = (long long)p.G * D2, NV = (long long)p.G * vdim;
  const bf16* kc = static_cast<const bf16*>(p.kcache) + (long long)p.tile_slot[tile] * p.cap * NK + g * D2;
  const bf16* vc = static_cast<const bf16*>(p.vcache) + (long long)p.tile_slot[tile] * p.cap * NV + g * vdim;
  const int kmin = chunk_start(p.tok_pos[row0 / rep], p.chunk), kmax = p.tok_pos[(row0 + rows - 1) / rep];
  const int n_kt = (kmax - kmin) / KT + 1, per = (n_kt + p.nsplit - 1) / p.nsplit;
  const int kt0 = split * per, kt1 = min(n_kt, kt0 + per);

  const int kw = D2 / 8, kdj = 128 / kw, kde = 128 - kdj * kw, kj0 = threadIdx.x / kw, ke0 = threadIdx.x - kj0 * kw;
  auto load_tile = [&](int kt, int buf) {
    const int kb = kmin + kt * KT, nk = min(KT, kmax + 1 - kb);
    bf16* K = Ks + buf * KT * QS;
    bf16* V = Vs + buf * KT * VS;
    const bf16* ksrc = kc + (long long)kb * NK;
    const bf16* vsrc = vc + (long long)kb * NV;
    // rows past the last key are zero, and so are value columns from vdim on; 16-byte chunk (row j, chunk e) by thread, stepping by 128
#pragma unroll 4
    for (int j = kj0, e = ke0; j < KT; ) {
      cp_async_16_or_zero(K + j * QS + e * 8, j < nk ? ksrc + j * (int)NK + e * 8 : kc, j < nk);
      j += kdj; e += kde;
      if (e >= kw) { e -= kw; ++j; }
    }
#pragma unroll
    for (int i = 0; i < KT * VT * 2 / 128; ++i) {
      const int c = threadIdx.x + i * 128, j = c / (VT * 2), e = (c % (VT * 2)) * 8;
      const bool ok = j < nk && e < vdim;
      cp_async_16_or_zero(V + j * VS + e, ok ? vsrc + j * (int)NV + e : vc, ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  {
    const int qw = D2 / 8;
    const bf16* q = static_cast<const bf16*>(p.q);
    for (int i = threadIdx.x; i < MR * qw; i += 128) {
      const int r = i / qw, e = (i - r * qw) * 8;
      const bool ok = r < rows;
      const int tok = (row0 + r) / rep;
      cp_async_16_or_zero(Qs + r * QS + e, ok ? q + (long long)tok * p.ldq + (long long)(g * rep + (row0 + r - tok * rep)) * D2 + e : q, ok);
    }
  }
  if (kt0 < kt1) load_tile(kt0, 0);
  else asm volatile("cp.async.commit_group;" ::: "memory");
  // the keys that this thread's two rows see
  const int wr = SK ? 0 : warp * 16;
  int lo[2], hi[2];
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int r = wr + g8 + 8 * hf;
    if (r < rows) { hi[hf] = p.tok_pos[(row0 + r) / rep]; lo[hf] = chunk_start(hi[hf], p.chunk); }
    else { hi[hf] = -1; lo[hf] = 0; }
  }
  // the bias rows of this thread's two heads, over distances
  const float* bh[2] = {nullptr, nullptr};
  if constexpr (NM == 1) {
    if (p.bias) {
      const float* table = p.bias + (long long)g * rep * (p.far + 1);
      if (p.bias_smem) {       // visible after the first tile's barrier
        float* bs = reinterpret_cast<float*>(smem_raw + p.bias_smem);
        for (int i = threadIdx.x; i < rep * (p.far + 1); i += 128) bs[i] = table[i];
        table = bs;
      }
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) bh[hf] = table + (long long)((row0 + wr + g8 + 8 * hf) % rep) * (p.far + 1);
    }
  }
  const int lo_last = chunk_start(kmax, p.chunk), pos_first = p.tok_pos[row0 / rep];      // a tile inside [lo_last, pos_first] is seen whole

  float o[NM][2 * VT][4];
  float rm[NM][2], rl[NM][2];       // [map][row half]
#pragma unroll
  for (int m = 0; m < NM; ++m) {
#pragma unroll
    for (int b = 0; b < 2 * VT; ++b) { o[m][b][0] = o[m][b][1] = o[m][b][2] = o[m][b][3] = 0.f; }
    rm[m][0] = rm[m][1] = -INFINITY; rl[m][0] = rl[m][1] = 0.f;
  }
  for (int kt = kt0, it = 0; kt < kt1; ++kt, ++it) {
    const int buf = it & 1;
    if (kt + 1 < kt1) { load_tile(kt + 1, buf ^ 1); asm volatile("cp.async.wait_group 1;" ::: "memory"); }
    else asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int wk = SK ? warp * 16 : 0;                 // this warp's first key of the tile
    const int kb = kmin + kt * KT + wk;
    const bf16* K = Ks + buf * KT * QS + wk * QS;
    const bf16* V = Vs + buf * KT * VS + wk * VS;
    const bool whole = kb >= lo_last && kb + NP * 16 - 1 <= pos_first;
    unsigned pf[NM][NP][4];
#pragma unroll
    for (int m = 0; m < NM; ++m) {
      float s[2 * NP][4];
#pragma unroll
      for (int b = 0; b < 2 * NP; ++b) { s[b][0] = s[b][1] = s[b][2] = s[b][3] = 0.f; }
      for (int ks = 0; ks < dim / 16; ++ks) {
        unsigned a[4];
        ldmatrix_x4(a, Qs + (wr + (mi & 1) * 8 + (lane & 7)) * QS + m * dim + ks * 16 + (mi >> 1) * 8);
#pragma unroll
        for (int np = 0; np < NP; ++np) {
          unsigned b[4];
          ldmatrix_x4(b, K + (np * 16 + (mi >> 1) * 8 + (lane & 7)) * QS + m * dim + ks * 16 + (mi & 1) * 8);
          mma_bf16_16816(s[2 * np], a, b[0], b[1]);
          mma_bf16_16816(s[2 * np + 1], a, b[2], b[3]);
        }
      }
      if constexpr (NM == 1) {
        if (p.bias) {
          if (pos_first - (kb + NP * 16 - 1) >= p.far) {      // every key of the tile is at least `far` back for every row
            const float b0 = bh[0][p.far], b1 = bh[1][p.far];
#pragma unroll
            for (int b = 0; b < 2 * NP; ++b) { s[b][0] += b0; s[b][1] += b0; s[b][2] += b1; s[b][3] += b1; }
          } else {
#pragma unroll
            for (int b = 0; b < 2 * NP; ++b)
#pragma unroll
              for (int e = 0; e < 4; ++e) s[b][e] += bh[e >> 1][min(max(hi[e >> 1] - (kb + b * 8 + 2 * t4 + (e & 1)), 0), p.far)];
          }
        }
      }
      if (!whole) {
#pragma unroll
        for (int b = 0; b < 2 * NP; ++b)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int j = kb + b * 8 + 2 * t4 + (e & 1);
            if (j < lo[e >> 1] || j > hi[e >> 1]) s[b][e] = -INFINITY;
          }
      }
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        float mx = -INFINITY;
#pragma unroll
        for (int b = 0; b < 2 * NP; ++b) mx = fmaxf(mx, fmaxf(s[b][2 * hf], s[b][2 * hf + 1]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float mn = fmaxf(rm[m][hf], mx), base = mn > -INFINITY ? mn * L2E : 0.f;
        const float corr = exp2_approx(rm[m][hf] * L2E - base);       // 0 before the first visible key
        rm[m][hf] = mn;
        float sum = 0.f;
#pragma unroll
        for (int b = 0; b < 2 * NP; ++b) {
          const float w0 = exp2_approx(fmaf(s[b][2 * hf], L2E, -base)), w1 = exp2_approx(fmaf(s[b][2 * hf + 1], L2E, -base));
          s[b][2 * hf] = w0; s[b][2 * hf + 1] = w1;
          sum += w0 + w1;
        }
        rl[m][hf] = rl[m][hf] * corr + sum;                     // this thread's share of the row's sum
        if (__any_sync(0xffffffffu, corr != 1.f)) {              // running maxima settle after a few tiles
#pragma unroll
          for (int b = 0; b < 2 * VT; ++b) { o[m][b][2 * hf] *= corr; o[m][b][2 * hf + 1] *= corr; }
        }
      }
#pragma unroll
      for (int np = 0; np < NP; ++np) {
        pf[m][np][0] = pack_bf16(s[2 * np][0], s[2 * np][1]);
        pf[m][np][1] = pack_bf16(s[2 * np][2], s[2 * np][3]);
        pf[m][np][2] = pack_bf16(s[2 * np + 1][0], s[2 * np + 1][1]);
        pf[m][np][3] = pack_bf16(s[2 * np + 1][2], s[2 * np + 1][3]);
      }
    }
#pragma unroll
    for (int np = 0; np < NP; ++np)
#pragma unroll
      for (int vt = 0; vt < VT; ++vt) {
        unsigned b[4];
        ldmatrix_x4_trans(b, V + (np * 16 + (mi & 1) * 8 + (lane & 7)) * VS + vt * 16 + (mi >> 1) * 8);
#pragma unroll
        for (int m = 0; m < NM; ++m) {
          mma_bf16_16816(o[m][2 * vt], pf[m][np], b[0], b[1]);
          mma_bf16_16816(o[m][2 * vt + 1], pf[m][np], b[2], b[3]);
        }
      }
    __syncthreads();
  }
#pragma unroll
  for (int m = 0; m < NM; ++m)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      rl[m][hf] += __shfl_xor_sync(0xffffffffu, rl[m][hf], 1);
      rl[m][hf] += __shfl_xor_sync(0xffffffffu, rl[m][hf], 2);
    }
  const int PSZ = NM * (vdim + 2);
  float* part = p.nsplit > 1 ? p.part + (((long long)tile * p.G + g) * p.nsplit + split) * MR * PSZ : nullptr;
  if constexpr (!SK) {
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int r = wr + g8 + 8 * hf;
      if (part) {
        if (r >= rows) continue;
        float* dst = part + (long long)r * PSZ;
#pragma unroll
        for (int m = 0; m < NM; ++m) {
#pragma unroll
          for (int b = 0; b < 2 * VT; ++b)
            if (b * 8 < vdim) *reinterpret_cast<float2*>(dst + m * vdim + b * 8 + 2 * t4) = make_float2(o[m][b][2 * hf], o[m][b][2 * hf + 1]);
          if (t4 == 0) { dst[NM * vdim + 2 * m] = rm[m][hf]; dst[NM * vdim + 2 * m + 1] = rl[m][hf]; }
        }
        continue;
      }
      if constexpr (NM == 1) {
        if (r >= rows) continue;
        const int tok = (row0 + r) / rep, head = g * rep + (row0 + r - tok * rep);
        const float i0 = rl[0][hf] > 0.f ? 1.f / rl[0][hf] : 0.f;
        bf16* out = static_cast<bf16*>(p.out) + (long long)tok * p.ldo + (long long)head * vdim;
        const bf16* eg = p.egate ? static_cast<const bf16*>(p.egate) + (long long)tok * p.lde + (long long)head * vdim : nullptr;
#pragma unroll
        for (int b = 0; b < 2 * VT; ++b)
          if (b * 8 < vdim) {
            float2 f = make_float2(i0, i0);
            if (eg) {
              const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(eg + b * 8 + 2 * t4));
              f.x *= sigmoidf(z.x); f.y *= sigmoidf(z.y);
            }
            *reinterpret_cast<unsigned*>(out + b * 8 + 2 * t4) = pack_bf16(o[0][b][2 * hf] * f.x, o[0][b][2 * hf + 1] * f.y);
          }
        continue;
      } else {
      // columns from vdim on are zero in both maps
      const float i0 = rl[0][hf] > 0.f ? 1.f / rl[0][hf] : 0.f, i1 = rl[NM - 1][hf] > 0.f ? p.lambda / rl[NM - 1][hf] : 0.f;
      float ss = 0.f;
#pragma unroll
      for (int b = 0; b < 2 * VT; ++b)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float v = o[0][b][2 * hf + e] * i0 - o[NM - 1][b][2 * hf + e] * i1;
          o[0][b][2 * hf + e] = v;
          ss = fmaf(v, v, ss);
        }
      ss += __shfl_xor_sync(0xffffffffu, ss, 1);
      ss += __shfl_xor_sync(0xffffffffu, ss, 2);
      if (r >= rows) continue;
      const int tok = (row0 + r) / rep, head = g * rep + (row0 + r - tok * rep);
      float f = p.out_scale / sqrtf(ss / (float)vdim + p.eps);
      if (p.gate) f *= sigmoidf(p.gate[(long long)tok * p.ldg + head]);
      bf16* out = static_cast<bf16*>(p.out) + (long long)tok * p.ldo + (long long)head * vdim;
#pragma unroll
      for (int b = 0; b < 2 * VT; ++b)
        if (b * 8 < vdim) *reinterpret_cast<unsigned*>(out + b * 8 + 2 * t4) = pack_bf16(o[0][b][2 * hf] * f, o[0][b][2 * hf + 1] * f);
      }
    }
  } else {
    // the warps' shares of the keys meet: every warp leaves its sums, then one warp per row weighs them
    constexpr int OS = VT * 16 + 4;
    asm volatile("cp.async.wait_group 0;" ::: "memory");         // the queries of a split without a key tile
    __syncthreads();
    float* mo = reinterpret_cast<float*>(smem_raw);               // [4 warps][NM maps][16 rows][OS]
    float* ml = mo + 4 * NM * 16 * OS;                            // [4][NM][16][2] maximum, sum
#pragma unroll
    for (int m = 0; m < NM; ++m)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int r = g8 + 8 * hf;
        if (r >= rows) continue;
        float* dst = mo + ((warp * NM + m) * 16 + r) * OS;
#pragma unroll
        for (int b = 0; b < 2 * VT; ++b) *reinterpret_cast<float2*>(dst + b * 8 + 2 * t4) = make_float2(o[m][b][2 * hf], o[m][b][2 * hf + 1]);
        if (t4 == 0) { float* d = ml + ((warp * NM + m) * 16 + r) * 2; d[0] = rm[m][hf]; d[1] = rl[m][hf]; }
      }
    __syncthreads();
    for (int r = warp; r < rows; r += 4) {
      float w[NM][4], M[NM], L[NM];
#pragma unroll
      for (int m = 0; m < NM; ++m) {
        M[m] = -INFINITY; L[m] = 0.f;
#pragma unroll
        for (int q = 0; q < 4; ++q) M[m] = fmaxf(M[m], ml[((q * NM + m) * 16 + r) * 2]);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float* d = ml + ((q * NM + m) * 16 + r) * 2;
          w[m][q] = d[0] > -INFINITY ? expf(d[0] - M[m]) : 0.f;
          L[m] += w[m][q] * d[1];
        }
      }
      auto sum = [&](int m, int c) {
        float a = 0.f;
#pragma unroll
        for (int q = 0; q < 4; ++q) a = fmaf(w[m][q], mo[((q * NM + m) * 16 + r) * OS + c], a);
        return a;
      };
      if (part) {
        float* dst = part + (long long)r * PSZ;
        for (int c = lane; c < vdim; c += 32) {
#pragma unroll
          for (int m = 0; m < NM; ++m) dst[m * vdim + c] = sum(m, c);
        }
#pragma unroll
        for (int m = 0; m < NM; ++m) if (lane == m) { dst[NM * vdim + 2 * m] = M[m]; dst[NM * vdim + 2 * m + 1] = L[m]; }
      } else {
        const float i0 = 1.f / L[0];
        if constexpr (NM == 1) {
          map_row_out<bf16, 1>(p, g, (long long)row0 + r, lane, [&](int c) { return sum(0, c) * i0; });
        } else {
          const float i1 = p.lambda / L[1];
          map_row_out<bf16, 2>(p, g, (long long)row0 + r, lane, [&](int c) { return sum(0, c) * i0 - sum(1, c) * i1; });
        }
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Router with groups, one warp per token: s = softmax(logits) over n outputs, or sigmoid(logits); choice score c = s + correction.
// n_groups > 1: only outputs of the `keep` groups (n / n_groups neighbours each) with the largest sum of their `group_sum` (1 or 2)
// largest choice scores may be chosen.  The `top` largest choice scores are chosen (ties: the lower index); their weights are s as
// it is, or (renorm) s / (sum of the chosen s + 1e-20) * out_scale.
// ---------------------------------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(128) moe_route_grouped_kernel(const float* __restrict__ logits, long long ldl, const float* __restrict__ correction, int n,
                                                                int top, int n_groups, int keep, int sigmoid, int group_sum, int renorm, float out_scale,
                                                                int* __restrict__ idx, float* __restrict__ wts, int n_tok) {
  extern __shared__ float route_buf[];      // per warp: [n] scores, [n] choice scores, [n_groups] group scores
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 4 + warp;
  if (t >= n_tok) return;
  float* s = route_buf + warp * (2 * n + n_groups);
  float* c = s + n;
  float* gs = c + n;
  const float* z = logits + (long long)t * ldl;
  float mx = -INFINITY, den = 0.f;
  if (sigmoid) {
    for (int e = lane; e < n; e += 32) s[e] = sigmoidf(z[e]);
    den = 1.f;
  } else {
    for (int e = lane; e < n; e += 32) mx = fmaxf(mx, z[e]);
    mx = warp_max(mx);
    for (int e = lane; e < n; e += 32) { const float w = expf(z[e] - mx); s[e] = w; den += w; }
    den = warp_sum(den);
  }
  __syncwarp();
  for (int e = lane; e < n; e += 32) { const float w = s[e] / den; s[e] = w; c[e] = w + correction[e]; }
  __syncwarp();
  // the largest entry of v[0 .. m), ties to the lower index; every lane gets it
  auto argmax = [&](const float* v, int m) {
    float best = -INFINITY; int bi = 0x7fffffff;
    for (int e = lane; e < m; e += 32) if (v[e] > best) { best = v[e]; bi = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o); const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    return bi;
  };
  if (n_groups > 1) {
    const int per = n / n_groups;
    for (int g = lane; g < n_groups; g += 32) {
      float b = -INFINITY, b2 = -INFINITY;       // the group's two largest
      for (int e = g * per; e < (g + 1) * per; ++e) { const float v = c[e]; if (v > b) { b2 = b; b = v; } else b2 = fmaxf(b2, v); }
      gs[g] = group_sum > 1 && per > 1 ? b + b2 : b;
    }
    __syncwarp();
    for (int k = 0; k < keep; ++k) {        // a kept group's score becomes NaN, which no comparison picks again
      const int g = argmax(gs, n_groups);
      __syncwarp();
      if (lane == 0 && g < n_groups) gs[g] = NAN;
      __syncwarp();
    }
    for (int e = lane; e < n; e += 32) if (!isnan(gs[e / per])) c[e] = -INFINITY;
    __syncwarp();
  }
  float sum = 0.f;
  for (int k = 0; k < top; ++k) {
    int e = argmax(c, n);
    if (e >= n) e = 0;                      // only when the logits are not finite
    sum += s[e];
    __syncwarp();
    if (lane == 0) { idx[(long long)t * top + k] = e; wts[(long long)t * top + k] = s[e]; c[e] = -INFINITY; }
    __syncwarp();
  }
  if (renorm && lane == 0)
    for (int k = 0; k < top; ++k) wts[(long long)t * top + k] *= out_scale / (sum + 1e-20f);
}

}  // namespace dlm
}  // namespace b200

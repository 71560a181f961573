// Further mechanisms of the decoder-LM handle (dlm.cu), first used by the Megolorn design: differential softmax attention on the
// query's own chunk of positions (two query / key maps per head over the same values), its query / key / value preparation with
// a bias, a norm per head and map and rotary positions, gated feed-forward units that share the preparation's launch, and a
// softmax router with a choice correction, groups and identity experts.
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

enum { GLU_CLAMPED = 0, GLU_SILU = 1 };
__device__ __forceinline__ float gated_unit(float g, float u, int kind, float limit) {
  return kind == GLU_CLAMPED ? clamped_gluf(g, u, limit) : g * sigmoidf(g) * u;
}

// ---------------------------------------------------------------------------------------------------------------------------
// Preparation of the attention and of the gated feed-forward beside it, on the concatenated projection proj T [tokens][ld].
// grid (tokens, head_rows + slices).  The first head_rows rows of the grid, one warp per (head, map): x + bias, / rms over dim * w (when w is given), rotated,
// queries times qscale -> qout TQ [tokens][Hm * dim], keys -> cache row (off_k < 0: the layer has no keys and values); values +
// bias -> cache row.  The rows after them: act[:, col] = gated_unit(proj[off_g + col], proj[off_u + col]) on GLU_SLICE columns each.
// ---------------------------------------------------------------------------------------------------------------------------
constexpr int GLU_SLICE = 2048;

struct DiffPrepParams {
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
  int off_g, off_u, F, glu; float limit;
  void* act; long long lda;             // T
  int head_rows;
};

template <typename T, typename TQ>
__global__ void __launch_bounds__(256) diff_prep_kernel(DiffPrepParams p) {
  extern __shared__ float prep_buf[];   // [8 warps][dim]
  const long long t = blockIdx.x;
  const T* row = static_cast<const T*>(p.proj) + t * p.ld;
  if ((int)blockIdx.y >= p.head_rows) {
    const int c0 = ((int)blockIdx.y - p.head_rows) * GLU_SLICE, c1 = min(p.F, c0 + GLU_SLICE);
    T* act = static_cast<T*>(p.act) + t * p.lda;
    if (sizeof(T) == 2 && ((p.F | p.off_g | p.off_u) & 7) == 0 && ((p.ld | p.lda) & 7) == 0 && ((uintptr_t)p.act & 15) == 0) {
      for (int c = c0 + threadIdx.x * 8; c < c1; c += 256 * 8) {
        const uint4 gv = *reinterpret_cast<const uint4*>(row + p.off_g + c), uv = *reinterpret_cast<const uint4*>(row + p.off_u + c);
        const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gv);
        const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&uv);
        uint4 ov;
        unsigned* o = reinterpret_cast<unsigned*>(&ov);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float2 g = __bfloat1622float2(g2[k]), u = __bfloat1622float2(u2[k]);
          o[k] = pack_bf16(gated_unit(g.x, u.x, p.glu, p.limit), gated_unit(g.y, u.y, p.glu, p.limit));
        }
        *reinterpret_cast<uint4*>(act + c) = ov;
      }
    } else {
      for (int c = c0 + threadIdx.x; c < c1; c += 256) act[c] = from_f<T>(gated_unit(to_f(row[p.off_g + c]), to_f(row[p.off_u + c]), p.glu, p.limit));
    }
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
      TQ* qo = static_cast<TQ*>(p.qout) + t * p.Hm * dim + i * dim;
      for (int e = lane; e < dim; e += 32) qo[e] = from_f<TQ>(rotary_at<float>(buf, e, p.half, p.adjacent, rot) * p.qscale);
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
// Differential attention.  Rows are (token, query head of ONE key/value head g) pairs, head fastest: row = token * rep + r,
// query head g * rep + r.  A tile is up to MR such rows of one request (tokens may be cut anywhere); every (tile, g) is a CTA of
// its own.  Per map m = 0, 1:  s_m[j] = q_m . k_m[j]  (q carries the scale),  lo <= j <= pos,  lo = start of pos's chunk (or 0);
// a_m = softmax(s_m) . V;   o = a_0 - lambda a_1;   out = o / sqrt(mean(o^2) + eps) * out_scale * sigmoid(gate).
// Cache rows: keys T [slots][cap][G][2][dim], values T [slots][cap][G][vdim].
// nsplit > 1 (grid.y): the key tiles are dealt over the splits, which leave per row [O_0 | O_1 | m_0 l_0 m_1 l_1] (sums of
// exp(s - m) v, running maximum, sum) for diff_attn_merge_kernel.
// ---------------------------------------------------------------------------------------------------------------------------
struct DiffAttnParams {
  const void* q; long long ldq;         // bf16 (tensor-core kernel) or fp32 [tokens][H][2][dim]
  const void *kcache, *vcache;
  const int *tile_row0, *tile_rows, *tile_slot, *tok_pos;
  const float* gate; long long ldg;     // [tokens][ldg] gate pre-activations, null: none
  void* out; long long ldo;             // T [tokens][ldo], head h at h * vdim
  float* part;                          // [tile][g][split][MR][2 * vdim + 4]
  int cap, H, G, dim, vdim, chunk, nsplit, n_tiles, MR, KT;
  float lambda, out_scale, eps;
};

__device__ __forceinline__ int chunk_start(int pos, int chunk) { return chunk > 0 ? pos / chunk * chunk : 0; }

// one row per warp: a0, a1 are the maps' results in shared or global memory; every lane calls
template <typename T, typename F>
__device__ __forceinline__ void diff_row_out(const DiffAttnParams& p, int g, long long row, int lane, F value) {
  const int rep = p.H / p.G;
  const long long tok = row / rep;
  const int head = g * rep + (int)(row - tok * rep);
  float ss = 0.f;
  for (int c = lane; c < p.vdim; c += 32) { const float o = value(c); ss = fmaf(o, o, ss); }
  float f = p.out_scale / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
  if (p.gate) f *= sigmoidf(p.gate[tok * p.ldg + head]);
  T* out = static_cast<T*>(p.out) + tok * p.ldo + (long long)head * p.vdim;
  for (int c = lane; c < p.vdim; c += 32) out[c] = from_f<T>(value(c) * f);
}

// CUDA cores, any sizes, fp32 arithmetic on T caches.  Shared memory: queries, accumulators, scores, staged keys and values.
inline size_t diff_attn_smem(int dim, int vdim, int MR, int KT) {
  return 4 * ((size_t)MR * 2 * dim + (size_t)MR * 2 * vdim + (size_t)MR * 2 * (KT + 1) + (size_t)3 * MR * 2 + (size_t)KT * (2 * dim + 1) + (size_t)KT * vdim);
}

template <typename T>
__global__ void __launch_bounds__(256) diff_attn_kernel(DiffAttnParams p) {
  extern __shared__ float da_smem[];
  const int dim = p.dim, vdim = p.vdim, MR = p.MR, KT = p.KT, rep = p.H / p.G, D2 = 2 * dim, KS = D2 + 1, SS = KT + 1;
  float* qs = da_smem;                                 // [MR][2][dim]
  float* oacc = qs + MR * D2;                          // [MR][2][vdim]
  float* sc = oacc + MR * 2 * vdim;                    // [MR][2][SS]
  float* rm = sc + MR * 2 * SS;                        // [MR][2] running maximum, sum, correction
  float* rl = rm + MR * 2;
  float* rc = rl + MR * 2;
  float* ks = rc + MR * 2;                             // [KT][KS]
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
  for (int i = threadIdx.x; i < MR * 2 * vdim; i += 256) oacc[i] = 0.f;
  for (int i = threadIdx.x; i < MR * 2; i += 256) { rm[i] = -INFINITY; rl[i] = 0.f; }
  for (int kt = kt0; kt < kt1; ++kt) {
    const int kb = kmin + kt * KT, nk = min(KT, kmax + 1 - kb);
    __syncthreads();
    for (int i = threadIdx.x; i < nk * D2; i += 256) { const int j = i / D2, e = i - j * D2; ks[j * KS + e] = to_f(kc[(long long)(kb + j) * p.G * D2 + e]); }
    for (int i = threadIdx.x; i < nk * vdim; i += 256) { const int j = i / vdim, e = i - j * vdim; vs[i] = to_f(vc[(long long)(kb + j) * p.G * vdim + e]); }
    __syncthreads();
    for (int i = threadIdx.x; i < rows * 2 * KT; i += 256) {      // scores, keys fastest
      const int rmi = i / KT, j = i - rmi * KT, r = rmi >> 1, m = rmi & 1;
      const int pos = p.tok_pos[(row0 + r) / rep];
      float s = -INFINITY;
      if (j < nk && kb + j <= pos && kb + j >= chunk_start(pos, p.chunk)) {
        const float *qv = qs + r * D2 + m * dim, *kv = ks + j * KS + m * dim;
        s = 0.f;
        for (int d = 0; d < dim; ++d) s = fmaf(qv[d], kv[d], s);
      }
      sc[rmi * SS + j] = s;
    }
    __syncthreads();
    for (int rmi = warp; rmi < rows * 2; rmi += 8) {              // online softmax, one warp per (row, map)
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
    for (int i = threadIdx.x; i < rows * 2 * vdim; i += 256) {
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
      const float *a0 = oacc + r * 2 * vdim, *a1 = a0 + vdim;
      const float i0 = 1.f / rl[2 * r], i1 = p.lambda / rl[2 * r + 1];
      diff_row_out<T>(p, g, row0 + r, lane, [&](int c) { return a0[c] * i0 - a1[c] * i1; });
    }
  } else {
    float* dst = p.part + (((long long)tile * p.G + g) * p.nsplit + split) * MR * (2 * vdim + 4);
    for (int i = threadIdx.x; i < rows * 2 * vdim; i += 256) { const int r = i / (2 * vdim); dst[(long long)r * (2 * vdim + 4) + (i - r * 2 * vdim)] = oacc[i]; }
    for (int i = threadIdx.x; i < rows * 2; i += 256) {
      float* d = dst + (long long)(i >> 1) * (2 * vdim + 4) + 2 * vdim + 2 * (i & 1);
      d[0] = rm[i]; d[1] = rl[i];
    }
  }
}

// merges the key splits, one warp per row; grid (tiles * G, rows / 4)
template <typename T>
__global__ void __launch_bounds__(128) diff_attn_merge_kernel(DiffAttnParams p) {
  const int tile = blockIdx.x / p.G, g = blockIdx.x % p.G, r = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= p.tile_rows[tile]) return;
  const int vdim = p.vdim, PS = 2 * vdim + 4;
  const float* base = p.part + (((long long)tile * p.G + g) * p.nsplit * p.MR + r) * PS;
  const long long ss = (long long)p.MR * PS;
  float f[2][2];       // lane s: weights of split s and s + 32 for the two maps
  for (int m = 0; m < 2; ++m) {
    const float ma = lane < p.nsplit ? base[lane * ss + 2 * vdim + 2 * m] : -INFINITY, la = lane < p.nsplit ? base[lane * ss + 2 * vdim + 2 * m + 1] : 0.f;
    const float mb = lane + 32 < p.nsplit ? base[(lane + 32) * ss + 2 * vdim + 2 * m] : -INFINITY, lb = lane + 32 < p.nsplit ? base[(lane + 32) * ss + 2 * vdim + 2 * m + 1] : 0.f;
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
    const float w0 = __shfl_sync(0xffffffffu, s < 32 ? f[0][0] : f[0][1], s & 31), w1 = __shfl_sync(0xffffffffu, s < 32 ? f[1][0] : f[1][1], s & 31);
    const float* src = base + s * ss;
#pragma unroll
    for (int i = 0; i < 32; ++i)
      if (lane + 32 * i < vdim) o[i] += w0 * src[lane + 32 * i] + w1 * src[vdim + lane + 32 * i];
  }
  const int rep = p.H / p.G;
  const long long row = p.tile_row0[tile] + r, tok = row / rep;
  const int head = g * rep + (int)(row - tok * rep);
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
inline size_t diff_attn_mma_smem(int dim, int VT, bool sk) {
  const size_t qs = 2 * dim + 8, vs = VT * 16 + 8, mr = sk ? 16 : 64;
  const size_t tiles = 2 * (mr * qs + 2 * DA_KT * qs + 2 * DA_KT * vs);
  const size_t meet = sk ? 4 * ((size_t)4 * 2 * 16 * (VT * 16 + 4) + 4 * 2 * 16 * 2) : 0;
  return std::max(tiles, meet);
}

template <int VT, bool SK>
__global__ void __launch_bounds__(128, 2) diff_attn_mma_kernel(DiffAttnParams p) {
  constexpr int MR = SK ? 16 : 64, KT = DA_KT, NP = SK ? 1 : 4, VS = VT * 16 + 8;
  constexpr float L2E = 1.4426950408889634f;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int dim = p.dim, vdim = p.vdim, rep = p.H / p.G, D2 = 2 * dim, QS = D2 + 8;
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
  const int lo_last = chunk_start(kmax, p.chunk), pos_first = p.tok_pos[row0 / rep];      // a tile inside [lo_last, pos_first] is seen whole

  float o[2][2 * VT][4];
  float rm[2][2], rl[2][2];       // [map][row half]
#pragma unroll
  for (int m = 0; m < 2; ++m) {
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
    unsigned pf[2][NP][4];
#pragma unroll
    for (int m = 0; m < 2; ++m) {
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
        for (int m = 0; m < 2; ++m) {
          mma_bf16_16816(o[m][2 * vt], pf[m][np], b[0], b[1]);
          mma_bf16_16816(o[m][2 * vt + 1], pf[m][np], b[2], b[3]);
        }
      }
    __syncthreads();
  }
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      rl[m][hf] += __shfl_xor_sync(0xffffffffu, rl[m][hf], 1);
      rl[m][hf] += __shfl_xor_sync(0xffffffffu, rl[m][hf], 2);
    }
  const int PSZ = 2 * vdim + 4;
  float* part = p.nsplit > 1 ? p.part + (((long long)tile * p.G + g) * p.nsplit + split) * MR * PSZ : nullptr;
  if constexpr (!SK) {
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int r = wr + g8 + 8 * hf;
      if (part) {
        if (r >= rows) continue;
        float* dst = part + (long long)r * PSZ;
#pragma unroll
        for (int m = 0; m < 2; ++m) {
#pragma unroll
          for (int b = 0; b < 2 * VT; ++b)
            if (b * 8 < vdim) *reinterpret_cast<float2*>(dst + m * vdim + b * 8 + 2 * t4) = make_float2(o[m][b][2 * hf], o[m][b][2 * hf + 1]);
          if (t4 == 0) { dst[2 * vdim + 2 * m] = rm[m][hf]; dst[2 * vdim + 2 * m + 1] = rl[m][hf]; }
        }
        continue;
      }
      // columns from vdim on are zero in both maps
      const float i0 = rl[0][hf] > 0.f ? 1.f / rl[0][hf] : 0.f, i1 = rl[1][hf] > 0.f ? p.lambda / rl[1][hf] : 0.f;
      float ss = 0.f;
#pragma unroll
      for (int b = 0; b < 2 * VT; ++b)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float v = o[0][b][2 * hf + e] * i0 - o[1][b][2 * hf + e] * i1;
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
  } else {
    // the warps' shares of the keys meet: every warp leaves its sums, then one warp per row weighs them
    constexpr int OS = VT * 16 + 4;
    asm volatile("cp.async.wait_group 0;" ::: "memory");         // the queries of a split without a key tile
    __syncthreads();
    float* mo = reinterpret_cast<float*>(smem_raw);               // [4 warps][2 maps][16 rows][OS]
    float* ml = mo + 4 * 2 * 16 * OS;                             // [4][2][16][2] maximum, sum
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int r = g8 + 8 * hf;
        if (r >= rows) continue;
        float* dst = mo + ((warp * 2 + m) * 16 + r) * OS;
#pragma unroll
        for (int b = 0; b < 2 * VT; ++b) *reinterpret_cast<float2*>(dst + b * 8 + 2 * t4) = make_float2(o[m][b][2 * hf], o[m][b][2 * hf + 1]);
        if (t4 == 0) { float* d = ml + ((warp * 2 + m) * 16 + r) * 2; d[0] = rm[m][hf]; d[1] = rl[m][hf]; }
      }
    __syncthreads();
    for (int r = warp; r < rows; r += 4) {
      float w[2][4], M[2], L[2];
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        M[m] = -INFINITY; L[m] = 0.f;
#pragma unroll
        for (int q = 0; q < 4; ++q) M[m] = fmaxf(M[m], ml[((q * 2 + m) * 16 + r) * 2]);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float* d = ml + ((q * 2 + m) * 16 + r) * 2;
          w[m][q] = d[0] > -INFINITY ? expf(d[0] - M[m]) : 0.f;
          L[m] += w[m][q] * d[1];
        }
      }
      auto sum = [&](int m, int c) {
        float a = 0.f;
#pragma unroll
        for (int q = 0; q < 4; ++q) a = fmaf(w[m][q], mo[((q * 2 + m) * 16 + r) * OS + c], a);
        return a;
      };
      if (part) {
        float* dst = part + (long long)r * PSZ;
        for (int c = lane; c < vdim; c += 32) { dst[c] = sum(0, c); dst[vdim + c] = sum(1, c); }
        if (lane < 2) { dst[2 * vdim + 2 * lane] = M[lane]; dst[2 * vdim + 2 * lane + 1] = L[lane]; }
      } else {
        const float i0 = 1.f / L[0], i1 = p.lambda / L[1];
        diff_row_out<bf16>(p, g, (long long)row0 + r, lane, [&](int c) { return sum(0, c) * i0 - sum(1, c) * i1; });
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// Softmax router, one warp per token: s = softmax(logits) over n outputs; choice score c = s + correction.  n_groups > 1: only
// outputs of the `keep` groups (n / n_groups neighbours each) with the largest single choice score may be chosen.  The `top`
// largest choice scores are chosen (ties: the lower index), their weights are s as it is.
// ---------------------------------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(128) moe_route_softmax_kernel(const float* __restrict__ logits, long long ldl, const float* __restrict__ correction, int n,
                                                                int top, int n_groups, int keep, int* __restrict__ idx, float* __restrict__ wts, int n_tok) {
  extern __shared__ float route_buf[];      // per warp: [n] scores, [n] choice scores, [n_groups] group scores
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 4 + warp;
  if (t >= n_tok) return;
  float* s = route_buf + warp * (2 * n + n_groups);
  float* c = s + n;
  float* gs = c + n;
  const float* z = logits + (long long)t * ldl;
  float mx = -INFINITY, den = 0.f;
  for (int e = lane; e < n; e += 32) mx = fmaxf(mx, z[e]);
  mx = warp_max(mx);
  for (int e = lane; e < n; e += 32) { const float w = expf(z[e] - mx); s[e] = w; den += w; }
  den = warp_sum(den);
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
      float b = -INFINITY;
      for (int e = g * per; e < (g + 1) * per; ++e) b = fmaxf(b, c[e]);
      gs[g] = b;
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
  for (int k = 0; k < top; ++k) {
    int e = argmax(c, n);
    if (e >= n) e = 0;                      // only when the logits are not finite
    __syncwarp();
    if (lane == 0) { idx[(long long)t * top + k] = e; wts[(long long)t * top + k] = s[e]; c[e] = -INFINITY; }
    __syncwarp();
  }
}

}  // namespace dlm
}  // namespace b200

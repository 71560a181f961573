// Further mechanisms of the decoder-LM handle (dlm.cu), first used by the Korirax design: a latent attention whose queries come
// through a latent too, the real-gated linear recurrence (RG-LRU: independent channels behind a short convolution, gates from
// block-diagonal products), and a per-layer token input behind every block.
//   T = activation / weight / cache type (bf16, or float in the all-fp32 mode).  Norms, positions and angles, the recurrence with
//   its gates, decays and state, and the residual stream are fp32 in both modes.
#pragma once

#include "dlm_mixers4.cuh"

namespace b200 {
namespace dlm {

// ---------------------------------------------------------------------------------------------------------------------------
// Latent attention with a query latent, preparation of both latents of a token and of the feed-forward beside it, on the
// concatenated projection proj T [tokens][ld].  grid (tokens, 1 + slices):
//   row 0:       cq[t] <- rms_norm(query latent) * wq;   cache row [rp] <- [ rms_norm(latent) * wc | rope(rotated key part) | zeros ]
//   other rows:  the feed-forward's unit on GLU_SLICE columns each
// ---------------------------------------------------------------------------------------------------------------------------
struct LatentPrepParams {
  const void* proj; long long ld;       // T
  int off_dq, q_rank, off_dkv, r, rd, rp, adjacent;
  const float *wq, *wc;
  void* cq; long long ldc;              // T
  void* cache; int cap;                 // T [slots][cap][rp]
  const float* rot;                     // [tokens][rd] cosines, sines
  const int *tok_slot, *tok_pos;
  float eps;
  UnitParams unit;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(LatentPrepParams p) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const T* row = static_cast<const T*>(p.proj) + t * p.ld;
  if (blockIdx.y > 0) {
    unit_slice<T>(p.unit, row, p.ld, t, ((int)blockIdx.y - 1) * GLU_SLICE);
    return;
  }
  if (p.q_rank > 0) {
    float s = 0.f;
    for (int i = threadIdx.x; i < p.q_rank; i += 256) { const float v = to_f(row[p.off_dq + i]); s = fmaf(v, v, s); }
    const float f = 1.f / sqrtf(block_sum(s, red) / (float)p.q_rank + p.eps);
    T* cq = static_cast<T*>(p.cq) + t * p.ldc;
    for (int i = threadIdx.x; i < p.q_rank; i += 256) cq[i] = from_f<T>(to_f(row[p.off_dq + i]) * f * p.wq[i]);
  }
  float s = 0.f;
  for (int i = threadIdx.x; i < p.r; i += 256) { const float v = to_f(row[p.off_dkv + i]); s = fmaf(v, v, s); }
  const float f = 1.f / sqrtf(block_sum(s, red) / (float)p.r + p.eps);
  T* dst = static_cast<T*>(p.cache) + ((long long)p.tok_slot[t] * p.cap + p.tok_pos[t]) * p.rp;
  for (int i = threadIdx.x; i < p.rp; i += 256) {
    float v = 0.f;
    if (i < p.r) v = to_f(row[p.off_dkv + i]) * f * p.wc[i];
    else if (i < p.r + p.rd) v = rotary_at(row + p.off_dkv + p.r, i - p.r, p.rd / 2, p.adjacent, p.rot + t * p.rd);
    dst[i] = from_f<T>(v);
  }
}

// qa[t][h][r .. r + rd) <- rope(rotated query part of head h) * scale, zeros up to rp (the first r elements are the query folded
// through W_uk, written by a product of its own); q T [tokens][ldq], H heads of [dim | rd]
template <typename T>
__global__ void __launch_bounds__(128) latent_query_rope_kernel(const T* __restrict__ q, long long ldq, int H, int dim, int rd, int r, int rp, int adjacent,
                                                                const float* __restrict__ rot, float scale, float* __restrict__ qa) {
  const long long t = blockIdx.x;
  const int tail = rp - r;
  for (int i = threadIdx.x; i < H * tail; i += 128) {
    const int hh = i / tail, d = i - hh * tail;
    qa[(t * H + hh) * rp + r + d] = d < rd ? rotary_at(q + t * ldq + hh * (dim + rd) + dim, d, rd / 2, adjacent, rot + t * rd) * scale : 0.f;
  }
}

// ---------------------------------------------------------------------------------------------------------------------------
// RG-LRU over C channels.  u = conv(px + bx) + bc (causal, `taps` taps, zeros in front of the sequence), gates r, i =
// sigmoid(block-diagonal products of u + biases), log a = lam8 r with lam8 = -8 softplus(lam),
//   S <- a S + sqrt(1 - a^2) i u   from S = 0,      out = S * gelu_tanh(py + by)
// The state [slots][C] is fp32 and carried between steps, like the convolution's last taps - 1 inputs (rows by position mod
// (taps - 1), bias included).
// ---------------------------------------------------------------------------------------------------------------------------
struct RgLruParams {
  const void* proj; long long ld;       // T [tokens][ld]
  int off_x, off_y, C, taps, bs;        // bs = channels of a gate matrix
  const float *bx, *by, *conv, *bc;     // conv [taps][C]
  float* hist;                          // [slots][taps - 1][C]
  float* u;                             // [tokens][C]
  const void* gates;                    // T [C / bs][2 bs][bs], rows 2c / 2c + 1 = r / i of the block's channel c
  const float *gate_b, *lam8;           // [2 C] interleaved, [C]
  float2* ab;                           // [tokens][C] (a, sqrt(1 - a^2) i u)
  float* state;                         // [slots][C]
  void* out; long long ldo;             // T
  const int *tok_slot, *tok_pos, *tok_first, *tok_last;
  const int *ent_tok0, *ent_ntok, *ent_slot, *ent_pos0;
  int n_tok;
  UnitParams unit;
  int conv_rows;
};

constexpr int CONV_SLICE = 512;

// grid (tokens / TT, conv_rows + slices): u on CONV_SLICE channels of TT neighbouring tokens each (many tokens: their loads overlap and
// share the taps); then the feed-forward's unit.  A token that is its request's only one in the step also puts its input into the
// carried rows (it alone reads them); conv_carry_kernel does so for longer portions.
template <typename T, int TT>
__global__ void __launch_bounds__(256) rglru_conv_kernel(RgLruParams p) {
  const long long t0 = (long long)blockIdx.x * TT;
  const int nt = TT == 1 ? 1 : (int)min((long long)TT, p.n_tok - t0);
  const T* row0 = static_cast<const T*>(p.proj) + t0 * p.ld;
  if ((int)blockIdx.y >= p.conv_rows) {
    for (int j = 0; j < nt; ++j) unit_slice<T>(p.unit, row0 + j * p.ld, p.ld, t0 + j, ((int)blockIdx.y - p.conv_rows) * GLU_SLICE);
    return;
  }
  const int keep = p.taps - 1, c1 = min(p.C, ((int)blockIdx.y + 1) * CONV_SLICE);
  // every tap of every token of the tile lies inside the step
  const bool inside = nt == TT && (int)t0 - p.tok_first[t0] >= keep && p.tok_last[t0] >= (int)t0 + TT - 1;
  for (int c = blockIdx.y * CONV_SLICE + threadIdx.x; c < c1; c += 256) {
    const float b = p.bx[c], bc = p.bc[c];
    const float* w = p.conv + c;
    const T* x = row0 + p.off_x + c;
    if (TT > 1 && inside) {
      float acc[TT];
      const float wk = w[(long long)keep * p.C];
#pragma unroll
      for (int j = 0; j < TT; ++j) acc[j] = fmaf(wk, to_f(x[j * p.ld]) + b, bc);
      for (int k = 1; k <= keep; ++k) {
        const float wv = w[(long long)(keep - k) * p.C];
#pragma unroll
        for (int j = 0; j < TT; ++j) acc[j] = fmaf(wv, to_f(x[(j - k) * p.ld]) + b, acc[j]);
      }
#pragma unroll
      for (int j = 0; j < TT; ++j) p.u[(t0 + j) * p.C + c] = acc[j];
      continue;
    }
    for (int j = 0; j < nt; ++j) {
      const long long t = t0 + j;
      const int pos = p.tok_pos[t], back = (int)t - p.tok_first[t];
      float* hist = p.hist + (long long)p.tok_slot[t] * keep * p.C;
      const float own = to_f(x[j * p.ld]) + b;
      float acc = fmaf(w[(long long)keep * p.C], own, bc);
      for (int k = 1; k <= keep && k <= pos; ++k) {
        const float v = k <= back ? to_f(x[(j - k) * p.ld]) + b : hist[(long long)((pos - k) % keep) * p.C + c];
        acc = fmaf(w[(long long)(keep - k) * p.C], v, acc);
      }
      p.u[t * p.C + c] = acc;
      if (keep > 0 && p.tok_first[t] == p.tok_last[t]) hist[(long long)(pos % keep) * p.C + c] = own;
    }
  }
}

__device__ __forceinline__ float2 rglru_coefficients(float zr, float zi, float lam8, float u) {
  const float la = lam8 * sigmoidf(zr);
  return make_float2(expf(la), sqrtf(-expm1f(2.f * la)) * sigmoidf(zi) * u);
}

// in place: raw gate products [tokens][C][2] -> (a, b)
__global__ void __launch_bounds__(256) rglru_coefficients_kernel(RgLruParams p) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= (long long)p.n_tok * p.C) return;
  const int c = (int)(i % p.C);
  const float2 z = p.ab[i];
  p.ab[i] = rglru_coefficients(z.x + p.gate_b[2 * c], z.y + p.gate_b[2 * c + 1], p.lam8[c], p.u[i]);
}

// one more token of a request: state and output
template <typename T>
__device__ __forceinline__ float rglru_output(const RgLruParams& p, long long t, int c, float S) {
  return S * gelu_tanhf(to_f(static_cast<const T*>(p.proj)[t * p.ld + p.off_y + c]) + p.by[c]);
}

// The gates' products on the tensor cores (mma.sync m16n8k16): u enters as the sum of two bf16 numbers, so that the products carry
// about 16 bits of u (the weights are bf16 as stored) into fp32 sums.  A thread holds r and i of a channel, and its epilogue leaves the
// recurrence's coefficients (STEP = false) or, when every request brings one token, takes the recurrence's step itself.
// bs a multiple of 16.  CTA: 64 tokens x 32 channels of one block; grid (2 bs / 64, tokens / 64, blocks).
template <bool STEP>
__global__ void __launch_bounds__(128) rglru_gates_mma_kernel(RgLruParams p) {
  constexpr int BK = 32, ST = BK + 8;
  __shared__ __align__(16) bf16 Ah[64][ST];
  __shared__ __align__(16) bf16 Al[64][ST];
  __shared__ __align__(16) bf16 Bs[64][ST];
  const int bs = p.bs, N = 2 * bs, m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const float* A = p.u + blockIdx.z * bs;
  const bf16* B = static_cast<const bf16*>(p.gates) + (long long)blockIdx.z * N * bs;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3, mi = lane >> 3;
  float acc[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i) { acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f; }
  float4 ra[4]; uint4 rb[2];
  auto fetch = [&](int k0) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = threadIdx.x + 128 * j, rr = c >> 3, kk = k0 + (c & 7) * 4;
      ra[j] = (m0 + rr < p.n_tok && kk < bs) ? *reinterpret_cast<const float4*>(A + (long long)(m0 + rr) * p.C + kk) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = threadIdx.x + 128 * j, rr = c >> 2, kk = k0 + (c & 3) * 8;
      rb[j] = (n0 + rr < N && kk < bs) ? *reinterpret_cast<const uint4*>(B + (long long)(n0 + rr) * bs + kk) : make_uint4(0u, 0u, 0u, 0u);
    }
  };
  fetch(0);
  for (int k0 = 0; k0 < bs; k0 += BK) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = threadIdx.x + 128 * j;
      const float v[4] = {ra[j].x, ra[j].y, ra[j].z, ra[j].w};
      float l[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) l[e] = v[e] - __bfloat162float(__float2bfloat16_rn(v[e]));
      *reinterpret_cast<uint2*>(&Ah[c >> 3][(c & 7) * 4]) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
      *reinterpret_cast<uint2*>(&Al[c >> 3][(c & 7) * 4]) = make_uint2(pack_bf16(l[0], l[1]), pack_bf16(l[2], l[3]));
    }
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int c = threadIdx.x + 128 * j;
      *reinterpret_cast<uint4*>(&Bs[c >> 2][(c & 3) * 8]) = rb[j];
    }
    __syncthreads();
    if (k0 + BK < bs) fetch(k0 + BK);
#pragma unroll
    for (int ks = 0; ks < BK / 16; ++ks) {
      unsigned ah[4], al[4];
      ldmatrix_x4(ah, &Ah[warp * 16 + (mi & 1) * 8 + (lane & 7)][ks * 16 + (mi >> 1) * 8]);
      ldmatrix_x4(al, &Al[warp * 16 + (mi & 1) * 8 + (lane & 7)][ks * 16 + (mi >> 1) * 8]);
#pragma unroll
      for (int np = 0; np < 4; ++np) {
        unsigned b[4];
        ldmatrix_x4(b, &Bs[np * 16 + (mi >> 1) * 8 + (lane & 7)][ks * 16 + (mi & 1) * 8]);
        mma_bf16_16816(acc[2 * np], al, b[0], b[1]);
        mma_bf16_16816(acc[2 * np + 1], al, b[2], b[3]);
        mma_bf16_16816(acc[2 * np], ah, b[0], b[1]);
        mma_bf16_16816(acc[2 * np + 1], ah, b[2], b[3]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int nb = 0; nb < 8; ++nb) {
    const int n = n0 + nb * 8 + 2 * t4;
    if (n >= N) continue;
    const int c = blockIdx.z * bs + (n >> 1);
    const float2 gb = *reinterpret_cast<const float2*>(p.gate_b + 2 * c);
    const float lam8 = p.lam8[c];
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int m = m0 + warp * 16 + g + 8 * hf;
      if (m >= p.n_tok) continue;
      const float2 ab = rglru_coefficients(acc[nb][2 * hf] + gb.x, acc[nb][2 * hf + 1] + gb.y, lam8, p.u[(long long)m * p.C + c]);
      if constexpr (STEP) {
        float* s = p.state + (long long)p.tok_slot[m] * p.C + c;
        const float S = p.tok_pos[m] > 0 ? fmaf(ab.x, *s, ab.y) : ab.y;
        *s = S;
        static_cast<bf16*>(p.out)[(long long)m * p.ldo + c] = __float2bfloat16_rn(rglru_output<bf16>(p, m, c, S));
      } else {
        p.ab[(long long)m * p.C + c] = ab;
      }
    }
  }
}

// The recurrence from its coefficients.  Block (channels, segments): a portion's tokens are cut into segments that run side by side:
// pass 1 leaves every segment's S_end = A S_start + B, every segment folds those in front of it into its start state, pass 2 walks
// again and writes the results.  Grid (ceil(C / channels), entries); dynamic shared memory 2 * channels * segments floats.
template <typename T>
__global__ void __launch_bounds__(1024, 1) rglru_scan_kernel(RgLruParams p) {
  extern __shared__ float seg_ab[];
  const int nx = blockDim.x, ns = blockDim.y, w = threadIdx.y, ent = blockIdx.y, c = blockIdx.x * nx + threadIdx.x;
  const bool live = c < p.C;
  const int tok0 = p.ent_tok0[ent], nt = p.ent_ntok[ent];
  const int len = (nt + ns - 1) / ns, t0 = min(nt, w * len), t1 = min(nt, t0 + len);
  const float2* ab = p.ab + (long long)tok0 * p.C + c;
  float a = 1.f, b = 0.f;
  if (live && ns > 1) {
#pragma unroll 8
    for (int i = t0; i < t1; ++i) {      // the loads do not depend on the state, so several tokens' loads may be in flight at once
      const float2 v = ab[(long long)i * p.C];
      b = fmaf(v.x, b, v.y);
      a *= v.x;
    }
  }
  seg_ab[2 * (w * nx + threadIdx.x)] = a; seg_ab[2 * (w * nx + threadIdx.x) + 1] = b;
  __syncthreads();
  if (!live) return;
  float* sp = p.state + (long long)p.ent_slot[ent] * p.C + c;
  float S = p.ent_pos0[ent] > 0 ? *sp : 0.f;
  for (int k = 0; k < w; ++k) S = fmaf(seg_ab[2 * (k * nx + threadIdx.x)], S, seg_ab[2 * (k * nx + threadIdx.x) + 1]);
#pragma unroll 8
  for (int i = t0; i < t1; ++i) {
    const float2 v = ab[(long long)i * p.C];
    S = fmaf(v.x, S, v.y);
    static_cast<T*>(p.out)[(long long)(tok0 + i) * p.ldo + c] = from_f<T>(rglru_output<T>(p, tok0 + i, c, S));
  }
  if (t1 == nt && t0 < t1) *sp = S;      // the segment that owns the portion's last token
}

// lam8 = -8 softplus(lam), once at load
__global__ void rglru_decay_kernel(const float* __restrict__ lam, float* __restrict__ lam8, int n) {
  const int i = blockIdx.x * 256 + threadIdx.x;
  if (i < n) lam8[i] = -8.f * (fmaxf(lam[i], 0.f) + log1pf(expf(-fabsf(lam[i]))));
}

// ---------------------------------------------------------------------------------------------------------------------------
// Per-layer token input: x <- x + rms_norm(W_proj (gelu_tanh(W_gate x) * e)) * w, e = a part of the token's row in a second table.
// ---------------------------------------------------------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ float side_entry(const T* __restrict__ table, long long ldt, int off, int id, int vocab, int d) {
  return id >= 0 && id < vocab ? to_f(table[(long long)id * ldt + off + d]) : 0.f;
}

// few tokens: gate product, GELU and the token's entry in one launch, from the fp32 residual; one warp per output, grid (tokens, dim / 8)
template <typename T>
__global__ void __launch_bounds__(256) side_gate_kernel(const float* __restrict__ xin, int W, const T* __restrict__ w, const T* __restrict__ table, long long ldt,
                                                        int off, const int* __restrict__ tokens, int vocab, int dim, T* __restrict__ out, long long ldo, int vec) {
  const long long t = blockIdx.x;
  const int d = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (d >= dim) return;
  const float* x = xin + t * W;
  const T* wr = w + (long long)d * W;
  float acc = 0.f;
  if (vec) {
#pragma unroll 4
    for (int k = lane * 8; k < W; k += 256) {
      float wv[8], xv[8];
      load8(wr + k, wv);
      load8(x + k, xv);
#pragma unroll
      for (int e = 0; e < 8; ++e) acc = fmaf(xv[e], wv[e], acc);
    }
  } else {
    for (int k = lane; k < W; k += 32) acc = fmaf(x[k], to_f(wr[k]), acc);
  }
  acc = warp_sum(acc);
  if (lane == 0) out[t * ldo + d] = from_f<T>(gelu_tanhf(acc) * side_entry(table, ldt, off, tokens[t], vocab, d));
}

// many tokens: what stands between the two products, in place on z T [tokens][ld]
template <typename T>
__global__ void __launch_bounds__(256) side_act_kernel(T* __restrict__ z, long long ld, const T* __restrict__ table, long long ldt, int off,
                                                       const int* __restrict__ tokens, int vocab, int dim, long long n) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  const long long t = i / dim; const int d = (int)(i - t * dim);
  z[t * ld + d] = from_f<T>(gelu_tanhf(to_f(z[t * ld + d])) * side_entry(table, ldt, off, tokens[t], vocab, d));
}

// x <- x + rms_norm(y) * w;  optional copy of x (per-layer trace);  x <- x + step (the vector in front of a pass, when given);
// optional h = rms_norm(x) * w_next.  One CTA per token.  REG (few tokens, W <= 4096): the row stays in registers.
template <typename T, bool REG>
__global__ void __launch_bounds__(256) side_end_kernel(float* __restrict__ xin, const T* __restrict__ y, const float* __restrict__ w, float* __restrict__ trace,
                                                       const float* __restrict__ step, const float* __restrict__ w_next, T* __restrict__ h, int W, float eps) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  float* x = xin + t * W;
  const T* yr = y + t * W;
  if constexpr (REG) {
    constexpr int NR = 16;
    float yv[NR], v[NR], s = 0.f;
#pragma unroll
    for (int k = 0; k < NR; ++k) {
      const int i = threadIdx.x + 256 * k;
      yv[k] = i < W ? to_f(yr[i]) : 0.f;
      v[k] = i < W ? x[i] : 0.f;
      s = fmaf(yv[k], yv[k], s);
    }
    const float f = 1.f / sqrtf(block_sum(s, red) / (float)W + eps);
    float q = 0.f;
#pragma unroll
    for (int k = 0; k < NR; ++k) {
      const int i = threadIdx.x + 256 * k;
      if (i >= W) break;
      v[k] += yv[k] * f * w[i];
      if (trace) trace[t * W + i] = v[k];
      if (step) v[k] += step[i];
      x[i] = v[k];
      q = fmaf(v[k], v[k], q);
    }
    if (!w_next) return;
    const float r = 1.f / sqrtf(block_sum(q, red) / (float)W + eps);
#pragma unroll
    for (int k = 0; k < NR; ++k) {
      const int i = threadIdx.x + 256 * k;
      if (i < W) h[t * W + i] = from_f<T>(v[k] * r * w_next[i]);
    }
    return;
  }
  float s = 0.f;
  for (int i = threadIdx.x; i < W; i += 256) { const float v = to_f(yr[i]); s = fmaf(v, v, s); }
  const float f = 1.f / sqrtf(block_sum(s, red) / (float)W + eps);
  float q = 0.f;
  for (int i = threadIdx.x; i < W; i += 256) {
    float v = x[i] + to_f(yr[i]) * f * w[i];
    if (trace) trace[t * W + i] = v;
    if (step) v += step[i];
    x[i] = v;
    q = fmaf(v, v, q);
  }
  if (!w_next) return;
  const float r = 1.f / sqrtf(block_sum(q, red) / (float)W + eps);
  for (int i = threadIdx.x; i < W; i += 256) h[t * W + i] = from_f<T>(x[i] * r * w_next[i]);
}

}  // namespace dlm
}  // namespace b200

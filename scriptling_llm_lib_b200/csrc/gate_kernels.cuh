// Kernels around gated mixers and gated side inputs, for float and bfloat16 activations (A):
//   qk_norm_store    biases of the projections, RMS norm of queries and keys (per head or over all heads, before they turn,
//                    or per head after),
//                    rotation by position, values mixed with an earlier layer's, queries out, keys and values into
//                    the paged cache
//   head_gate        attention output of every head times the sigmoid of that head's gate logit
//   add_cast         residual stream += pending addend; a copy of the stream in the element type
//   gelu_mul_rows    gelu(a) times a slice of a per-token table row
//   add_rms_normed   residual stream += y / rms(y) * w
//   softcap          cap * tanh(x / cap) in place
// Norms, sums of squares, angles, sigmoids and the residual sum are float whatever A is.
#pragma once
#include "common.cuh"

namespace gate {

template <typename A> __device__ __forceinline__ float ld_flag(const void* p, int is_f32, size_t i) {
  return is_f32 ? ((const float*)p)[i] : to_f32(((const A*)p)[i]);
}
__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float gelu_tanh_f(float v) {
  return 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
}

// ------------------------------------------------------------------ biases, query/key norm, rotation, value mixing, cache write
// Row t of c (float or A, row stride ld) holds [H query heads of hd | G key heads of hd | G value heads of vd], to which
// `bias` (float, the same columns, or null) is added first. With qw / kw (norm weights; either may be null) queries and
// keys are divided by their root mean square and multiplied by the weight: over ALL the columns of the query part and of
// the key part (weights of H * hd and G * hd), or with `per_head` over every head by itself (weights of hd, shared by the
// heads). Then the first `rot` dims of every query and key head turn by the token's position (table cs[pos][i] = (cos, sin);
// half pairing i with i + rot / 2, or adjacent pairs). With `norm_after` every query and key head is instead divided by its
// root mean square once it has turned, without a weight (qw and kw null). Queries go to q_out [T, ldq], keys and values to the token's place in
// the cache pages. Values may be mixed on the way with those an earlier layer projected for the same token, kept in vmix
// [T, G * vd]: mix_mode 1 writes them there, mode 2 stores (1 - lam) * v + lam * vmix. G == 0: queries only.
struct QkStoreArgs {
  const void* c; int c_f32; int ld;
  const float* bias;
  void* q_out; int ldq;
  const int* tok_pos; const int* tok_seq; const int* block_table; int max_pages;
  const float2* cs;
  void* kpages; void* vpages;
  int H, G, hd, vd, rot, interleaved;
  const void* qw; const void* kw; int w_f32; int per_head; float eps;
  void* vmix; int mix_mode; float lam;
  int norm_after;
};

template <int V> struct Pack { float f[V]; };
template <int V> __device__ __forceinline__ Pack<V> ld_pack(const float* p) {
  Pack<V> r;
  if constexpr (V == 4) { float4 v = *(const float4*)p; r.f[0] = v.x; r.f[1] = v.y; r.f[2] = v.z; r.f[3] = v.w; }
  else r.f[0] = *p;
  return r;
}
template <int V> __device__ __forceinline__ Pack<V> ld_pack(const bf16* p) {
  Pack<V> r;
  if constexpr (V == 4) { float4 v = ld4(p); r.f[0] = v.x; r.f[1] = v.y; r.f[2] = v.z; r.f[3] = v.w; }
  else r.f[0] = to_f32(*p);
  return r;
}
template <typename A, int V> __device__ __forceinline__ Pack<V> ld_pack_flag(const void* p, int is_f32, size_t i) {
  return is_f32 ? ld_pack<V>((const float*)p + i) : ld_pack<V>((const A*)p + i);
}
template <typename A, int V> __device__ __forceinline__ void st_pack(A* p, const Pack<V>& r) {
  if constexpr (V == 4) st4(p, make_float4(r.f[0], r.f[1], r.f[2], r.f[3]));
  else *p = from_f32<A>(r.f[0]);
}

#define QKS_WARPS 8
// V elements a lane and access (4 where widths and addresses allow, else 1), NIT accesses to a head. A warp takes NB heads at
// a time, whose loads are all asked for before the first is used and whose elements stay in registers up to the stores; with
// a norm over the whole projection they stay over the block's two sums as well where one such batch a warp covers all heads.
template <typename A, int V, int NIT, int NB>
__global__ void __launch_bounds__(QKS_WARPS * 32) qk_norm_store_kernel(QkStoreArgs p) {
  __shared__ float red[2][QKS_WARPS];
  extern __shared__ float qks_row[];             // with a rotation: hd floats a warp
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int H = p.H, heads = p.H + p.G, hd = p.hd, vd = p.vd, QW = H * hd, KW = p.G * hd, VW = p.G * vd;
  const int pos = p.tok_pos[t];
  const size_t row = (size_t)t * p.ld;
  size_t page_slot = 0;
  if (p.G > 0) {
    int page = p.block_table[(size_t)p.tok_seq[t] * p.max_pages + pos / SLLM_PAGE];
    page_slot = (size_t)page * p.G * SLLM_PAGE + (pos % SLLM_PAGE);     // + g * PAGE, times the head width
  }
  // the block's first values are on their way while queries and keys are worked
  const int e0 = threadIdx.x * V;
  Pack<V> val;
  if (e0 < VW) val = ld_pack_flag<A, V>(p.c, p.c_f32, row + QW + KW + e0);

  Pack<V> x[NB][NIT];
  auto load = [&](int first) {                   // heads first, first + QKS_WARPS, ...
#pragma unroll
    for (int n = 0; n < NB; n++) {
      const int head = first + n * QKS_WARPS;
#pragma unroll
      for (int it = 0; it < NIT; it++) {
        const int j = (it * 32 + lane) * V;
        if (head < heads && j < hd) x[n][it] = ld_pack_flag<A, V>(p.c, p.c_f32, row + head * hd + j);
      }
    }
    if (p.bias) {
#pragma unroll
      for (int n = 0; n < NB; n++) {
        const int head = first + n * QKS_WARPS;
#pragma unroll
        for (int it = 0; it < NIT; it++) {
          const int j = (it * 32 + lane) * V;
          if (head < heads && j < hd) {
            const Pack<V> b = ld_pack<V>(p.bias + head * hd + j);
#pragma unroll
            for (int i = 0; i < V; i++) x[n][it].f[i] += b.f[i];
          }
        }
      }
    }
  };
  auto squares = [&](int n, int head) -> float {  // this lane's share of a head's sum
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < NIT; it++)
      if (head < heads && (it * 32 + lane) * V < hd) {
#pragma unroll
        for (int i = 0; i < V; i++) ss = fmaf(x[n][it].f[i], x[n][it].f[i], ss);
      }
    return ss;
  };
  constexpr int BATCH = QKS_WARPS * NB;
  const bool whole = !p.per_head && (p.qw || p.kw);
  float rq = 1.f, rk = 1.f;
  if (whole) {
    float sq = 0.f, sk = 0.f;
    for (int first = warp; first < heads; first += BATCH) {
      load(first);
#pragma unroll
      for (int n = 0; n < NB; n++) {
        const int head = first + n * QKS_WARPS;
        const float ss = squares(n, head);
        if (head < H) sq += ss; else sk += ss;
      }
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < QKS_WARPS; w++) { sq += red[0][w]; sk += red[1][w]; }
    if (p.qw) rq = 1.0f / sqrtf(sq / (float)QW + p.eps);
    if (p.kw && KW > 0) rk = 1.0f / sqrtf(sk / (float)KW + p.eps);
  }
  const int half = p.rot >> 1;
  const float2* csr = p.cs + (size_t)pos * half;
  float* wrow = qks_row + warp * hd;
  for (int first = warp; first < heads; first += BATCH) {
    if (!(whole && heads <= BATCH)) load(first);
#pragma unroll
    for (int n = 0; n < NB; n++) {
      const int head = first + n * QKS_WARPS;
      if (head >= heads) break;
      const bool is_q = head < H;
      const int col = head * hd;                                         // the key part follows the query part directly
      const void* w = is_q ? p.qw : p.kw;
      const int wc = p.per_head ? 0 : is_q ? col : col - QW;
      float r = is_q ? rq : rk;
      if (p.per_head && w) r = 1.0f / sqrtf(warp_sum(squares(n, head)) / (float)hd + p.eps);
      A* dst = is_q ? (A*)p.q_out + (size_t)t * p.ldq + col : (A*)p.kpages + (page_slot + (size_t)(head - H) * SLLM_PAGE) * hd;
      if constexpr (V == 4) {
        if (p.norm_after && (p.interleaved || p.rot == 0)) {             // a lane's four elements are two whole pairs: no exchange
#pragma unroll
          for (int it = 0; it < NIT; it++) {
            const int j = (it * 32 + lane) * V;
#pragma unroll
            for (int i = 0; i < V; i += 2)
              if (j + i < p.rot) {
                const float2 a = csr[(j + i) >> 1];
                const float x0 = x[n][it].f[i], x1 = x[n][it].f[i + 1];
                x[n][it].f[i] = x0 * a.x - x1 * a.y;
                x[n][it].f[i + 1] = x1 * a.x + x0 * a.y;
              }
          }
          r = 1.0f / sqrtf(warp_sum(squares(n, head)) / (float)hd + p.eps);
#pragma unroll
          for (int it = 0; it < NIT; it++) {
            const int j = (it * 32 + lane) * V;
            if (j >= hd) break;
#pragma unroll
            for (int i = 0; i < V; i++) x[n][it].f[i] *= r;
            st_pack<A, V>(dst + j, x[n][it]);
          }
          continue;
        }
      }
      if (p.norm_after && p.rot == 0) {
        r = 1.0f / sqrtf(warp_sum(squares(n, head)) / (float)hd + p.eps);
#pragma unroll
        for (int it = 0; it < NIT; it++)
          if ((it * 32 + lane) * V < hd) {
#pragma unroll
            for (int i = 0; i < V; i++) x[n][it].f[i] *= r;
          }
      }
#pragma unroll
      for (int it = 0; it < NIT; it++) {
        const int j = (it * 32 + lane) * V;
        if (j >= hd) break;
        if (w) {
          const Pack<V> ww = ld_pack_flag<bf16, V>(w, p.w_f32, wc + j);
#pragma unroll
          for (int i = 0; i < V; i++) x[n][it].f[i] = x[n][it].f[i] * r * ww.f[i];
        }
        if (p.rot > 0) {
#pragma unroll
          for (int i = 0; i < V; i++) wrow[j + i] = x[n][it].f[i];
        } else {
          st_pack<A, V>(dst + j, x[n][it]);
        }
      }
      if (p.rot > 0) {                                                   // a lane turns a pair; the rest passes as it is
        __syncwarp();
        float ra = 1.f;
        if (p.norm_after) {                                              // the sum is over the turned head
          float ss = 0.f;
          for (int i = lane; i < half; i += 32) {
            const int i0 = p.interleaved ? 2 * i : i, i1 = p.interleaved ? 2 * i + 1 : i + half;
            const float2 a = csr[i];
            const float x0 = wrow[i0], x1 = wrow[i1], y0 = x0 * a.x - x1 * a.y, y1 = x1 * a.x + x0 * a.y;
            ss = fmaf(y0, y0, fmaf(y1, y1, ss));
          }
          for (int j = p.rot + lane; j < hd; j += 32) ss = fmaf(wrow[j], wrow[j], ss);
          ra = 1.0f / sqrtf(warp_sum(ss) / (float)hd + p.eps);
        }
        for (int i = lane; i < half; i += 32) {
          const int i0 = p.interleaved ? 2 * i : i, i1 = p.interleaved ? 2 * i + 1 : i + half;
          const float2 a = csr[i];
          const float x0 = wrow[i0], x1 = wrow[i1];
          dst[i0] = from_f32<A>((x0 * a.x - x1 * a.y) * ra);
          dst[i1] = from_f32<A>((x1 * a.x + x0 * a.y) * ra);
        }
        for (int j = p.rot + lane; j < hd; j += 32) dst[j] = from_f32<A>(wrow[j] * ra);
        __syncwarp();
      }
    }
  }
  // values, the block over all heads
  A* vm = (A*)p.vmix + (size_t)t * VW;
  for (int e = e0; e < VW; e += QKS_WARPS * 32 * V) {
    const int g = e / vd, j = e % vd;
    if (e != e0) val = ld_pack_flag<A, V>(p.c, p.c_f32, row + QW + KW + e);
    if (p.bias) {
      const Pack<V> b = ld_pack<V>(p.bias + QW + KW + e);
#pragma unroll
      for (int i = 0; i < V; i++) val.f[i] += b.f[i];
    }
    if (p.mix_mode == 1) st_pack<A, V>(vm + e, val);
    if (p.mix_mode == 2) {
      const Pack<V> f = ld_pack<V>((const A*)vm + e);
#pragma unroll
      for (int i = 0; i < V; i++) val.f[i] = (1.0f - p.lam) * val.f[i] + p.lam * f.f[i];
    }
    st_pack<A, V>((A*)p.vpages + (page_slot + (size_t)g * SLLM_PAGE) * vd + j, val);
  }
}

// The common case of the above (heads of up to 128 in multiples of 4, at most 8 NB query and key heads, float weights; no
// rotation, or with ROT adjacent pairs: a lane's four elements are two whole pairs, whose angles it reads once for all heads;
// BARE: neither biases nor weights nor mixed values, which leaves room for more warps): a
// warp's heads in one batch, and every load is asked for before the first is used; biases and weights, which no kernel of a
// step writes, even before the wait for the kernel in front.
__device__ __forceinline__ float4 turned(const float4& x, const float2& a, const float2& b) {
  return make_float4(x.x * a.x - x.y * a.y, x.y * a.x + x.x * a.y, x.z * b.x - x.w * b.y, x.w * b.x + x.z * b.y);
}
template <typename A, int NB, bool ROT, bool BARE>
__global__ void __launch_bounds__(QKS_WARPS * 32) qk_norm_store_small_kernel(QkStoreArgs p) {
  __shared__ float red[2][QKS_WARPS];
  pdl_launch_dependents();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, j = (threadIdx.x & 31) * 4;
  const int H = p.H, heads = p.H + p.G, hd = p.hd, QW = H * hd, KW = p.G * hd, VW = p.G * p.vd;
  const bool on = j < hd;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 b[NB], w[NB], x[NB];
#pragma unroll
  for (int n = 0; n < NB; n++) {
    const int head = warp + n * QKS_WARPS;
    const bool ok = on && head < heads;
    const float* wp = (const float*)(head < H ? p.qw : p.kw);
    b[n] = !BARE && ok && p.bias ? *(const float4*)(p.bias + head * hd + j) : zero;
    w[n] = !BARE && ok && wp ? *(const float4*)(wp + (p.per_head ? j : head < H ? head * hd + j : head * hd - QW + j)) : zero;
  }
  const int e = threadIdx.x * 4;
  float4 vb = !BARE && p.bias && e < VW ? *(const float4*)(p.bias + QW + KW + e) : zero;
  pdl_wait();
  const int pos = p.tok_pos[t];
  const A* c = (const A*)p.c + (size_t)t * p.ld;
  A* vm = (A*)p.vmix + (size_t)t * VW;
#pragma unroll
  for (int n = 0; n < NB; n++) x[n] = on && warp + n * QKS_WARPS < heads ? ld4(c + (warp + n * QKS_WARPS) * hd + j) : zero;
  float2 r0 = make_float2(1.f, 0.f), r1 = r0;    // (cos, sin) of the lane's pairs; those behind the rotated dims stay as they are
  if constexpr (ROT) {
    const float2* csr = p.cs + (size_t)pos * (p.rot >> 1) + (j >> 1);
    if (j < p.rot) r0 = csr[0];
    if (j + 2 < p.rot) r1 = csr[1];
  }
  float4 v = e < VW ? ld4(c + QW + KW + e) : zero, f = !BARE && p.mix_mode == 2 && e < VW ? ld4((const A*)vm + e) : zero;
  size_t page_slot = 0;
  if (p.G > 0) {
    const int page = p.block_table[(size_t)p.tok_seq[t] * p.max_pages + pos / SLLM_PAGE];
    page_slot = (size_t)page * p.G * SLLM_PAGE + (pos % SLLM_PAGE);
  }
  float ss[NB];
#pragma unroll
  for (int n = 0; n < NB; n++) {
    if (!BARE) { x[n].x += b[n].x; x[n].y += b[n].y; x[n].z += b[n].z; x[n].w += b[n].w; }
    if (ROT && p.norm_after) x[n] = turned(x[n], r0, r1);
    ss[n] = warp_sum(fmaf(x[n].x, x[n].x, fmaf(x[n].y, x[n].y, fmaf(x[n].z, x[n].z, x[n].w * x[n].w))));
  }
  float rq = 1.f, rk = 1.f;
  if (!BARE && !p.per_head && (p.qw || p.kw)) {
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int n = 0; n < NB; n++) {
      if (warp + n * QKS_WARPS < H) sq += ss[n]; else sk += ss[n];
    }
    if (j == 0) { red[0][warp] = sq; red[1][warp] = sk; }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < QKS_WARPS; i++) { sq += red[0][i]; sk += red[1][i]; }
    rq = 1.0f / sqrtf(sq / (float)QW + p.eps);
    rk = 1.0f / sqrtf(sk / (float)(KW > 0 ? KW : 1) + p.eps);
  }
#pragma unroll
  for (int n = 0; n < NB; n++) {
    const int head = warp + n * QKS_WARPS;
    if (head < heads && on) {
      if (!BARE && (head < H ? p.qw != nullptr : p.kw != nullptr)) {
        const float r = p.per_head ? 1.0f / sqrtf(ss[n] / (float)hd + p.eps) : head < H ? rq : rk;
        x[n] = make_float4(x[n].x * r * w[n].x, x[n].y * r * w[n].y, x[n].z * r * w[n].z, x[n].w * r * w[n].w);
      } else if (p.norm_after) {
        const float r = 1.0f / sqrtf(ss[n] / (float)hd + p.eps);
        x[n] = make_float4(x[n].x * r, x[n].y * r, x[n].z * r, x[n].w * r);
      }
      if (ROT && !p.norm_after) x[n] = turned(x[n], r0, r1);
      if (head < H) st4((A*)p.q_out + (size_t)t * p.ldq + head * hd + j, x[n]);
      else st4((A*)p.kpages + (page_slot + (size_t)(head - H) * SLLM_PAGE) * hd + j, x[n]);
    }
  }
  for (int k = e; k < VW; k += QKS_WARPS * 32 * 4) {
    if (k != e) {
      v = ld4(c + QW + KW + k);
      if (!BARE && p.bias) vb = *(const float4*)(p.bias + QW + KW + k);
      if (!BARE && p.mix_mode == 2) f = ld4((const A*)vm + k);
    }
    if (!BARE) { v.x += vb.x; v.y += vb.y; v.z += vb.z; v.w += vb.w; }
    if (!BARE && p.mix_mode == 1) st4(vm + k, v);
    if (!BARE && p.mix_mode == 2) {
      const float a = 1.0f - p.lam;
      v = make_float4(a * v.x + p.lam * f.x, a * v.y + p.lam * f.y, a * v.z + p.lam * f.z, a * v.w + p.lam * f.w);
    }
    st4((A*)p.vpages + (page_slot + (size_t)(k / p.vd) * SLLM_PAGE) * p.vd + k % p.vd, v);
  }
}

// ------------------------------------------------------------------ convolution, norm, rotation, cache write
// The same as qk_norm_store behind a short causal convolution, one block a token and the row never leaving the
// chip: row t of y (A, row stride ldy) is the projection [queries | keys | values] of C = (H + G) hd + G vd
// columns; c[t][ch] = sum_j cw[ch][j] * y[t - taps + 1 + j][ch], rows before the step's first one of the sequence
// coming from its state [slot][taps - 1][C] (float, oldest first). c is kept as floats in shared memory, the sums
// of squares are taken on the way, then norm, rotation and stores as above. `own_state`: every sequence has one
// row in the step, and the block moves the sequence's state on by itself (a channel's entries are read and
// written by one thread); otherwise conv_state_kernel follows.
struct ConvNormArgs {
  const void* y; int ldy;
  const void* cw; int cw_f32; int taps;
  float* state; const int* seq_start; const int* tok_seq; const int* slots; int own_state;
  void* q_out; int ldq;
  const int* tok_pos; const int* block_table; int max_pages; const float2* cs;
  void* kpages; void* vpages;
  int H, G, hd, vd, rot, interleaved;
  const void* qw; const void* kw; int w_f32; float eps;
};

__device__ __forceinline__ void st2(float* p, float a, float b) { *(float2*)p = make_float2(a, b); }
__device__ __forceinline__ void st2(bf16* p, float a, float b) { *(__nv_bfloat162*)p = __floats2bfloat162_rn(a, b); }

template <typename A> __device__ __forceinline__ float4 ld4f(const void* p, int is_f32, size_t i) {
  return is_f32 ? ld4((const float*)p + i) : ld4((const A*)p + i);
}

// Four channels from c on with a number of taps known to the compiler: every load is issued before the first sum.
template <typename A, int TAPS>
__device__ __forceinline__ float4 conv_four(const ConvNormArgs& p, const A* __restrict__ y, float* st, int t, int first, int C, int c) {
  constexpr int HIST = TAPS - 1;
  float4 v[TAPS];
  float w[4 * TAPS];                           // the four channels' taps lie one behind the other
#pragma unroll
  for (int j = 0; j < TAPS; j++) {
    int s = t - HIST + j;
    v[j] = s >= first ? ld4(y + (size_t)s * p.ldy + c) : *(const float4*)(st + (size_t)(HIST + (s - first)) * C + c);
  }
#pragma unroll
  for (int m = 0; m < TAPS; m++) {
    float4 q = ld4f<A>(p.cw, p.cw_f32, (size_t)c * TAPS + 4 * m);
    w[4 * m] = q.x; w[4 * m + 1] = q.y; w[4 * m + 2] = q.z; w[4 * m + 3] = q.w;
  }
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < TAPS; j++) {
    acc.x += w[j] * v[j].x;
    acc.y += w[TAPS + j] * v[j].y;
    acc.z += w[2 * TAPS + j] * v[j].z;
    acc.w += w[3 * TAPS + j] * v[j].w;
  }
  if (p.own_state) {
#pragma unroll
    for (int j = 1; j < TAPS; j++) *(float4*)(st + (size_t)(j - 1) * C + c) = v[j];
  }
  return acc;
}

// VEC: four channels a thread. TAPS: the number of taps where the compiler knows it (VEC only), 0: p.taps.
template <typename A, int VEC, int TAPS>
__global__ void __launch_bounds__(256, 5) conv_qk_norm_store_kernel(ConvNormArgs p) {
  extern __shared__ __align__(16) float crow[];
  __shared__ float red[32];
  const A* y = (const A*)p.y;
  int t = blockIdx.x;
  int b = p.tok_seq[t];                        // the row's indices first, all at once: the stores below keep loads behind them
  int pos = p.tok_pos[t];
  int first = p.seq_start[b];
  int slot = p.slots[b];
  int page = p.G > 0 ? p.block_table[(size_t)b * p.max_pages + pos / SLLM_PAGE] : 0;
  int hist = p.taps - 1;
  int QW = p.H * p.hd, KW = p.G * p.hd, C = QW + KW + p.G * p.vd;
  float* st = p.state + (size_t)slot * hist * C;
  float ssq = 0.f, ssk = 0.f;
  if (VEC) {                                   // four channels a thread: C, QW, KW, ldy multiples of four
    for (int c = threadIdx.x * 4; c < C; c += blockDim.x * 4) {
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      if (TAPS > 0) acc = conv_four<A, TAPS ? TAPS : 1>(p, y, st, t, first, C, c);
      else
      for (int j = 0; j < p.taps; j++) {
        int s = t - hist + j;
        float4 v = s >= first ? ld4(y + (size_t)s * p.ldy + c) : *(const float4*)(st + (size_t)(hist + (s - first)) * C + c);
        acc.x += load_w(p.cw, p.cw_f32, (size_t)c * p.taps + j) * v.x;
        acc.y += load_w(p.cw, p.cw_f32, (size_t)(c + 1) * p.taps + j) * v.y;
        acc.z += load_w(p.cw, p.cw_f32, (size_t)(c + 2) * p.taps + j) * v.z;
        acc.w += load_w(p.cw, p.cw_f32, (size_t)(c + 3) * p.taps + j) * v.w;
        if (p.own_state && j > 0) *(float4*)(st + (size_t)(j - 1) * C + c) = v;      // entry j moves to j - 1
      }
      *(float4*)(crow + c) = acc;
      float q = acc.x * acc.x + acc.y * acc.y + acc.z * acc.z + acc.w * acc.w;
      if (c < QW) ssq += q; else if (c < QW + KW) ssk += q;
    }
  } else {
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
      float acc = 0.f;
      for (int j = 0; j < p.taps; j++) {
        int s = t - hist + j;
        float v = s >= first ? to_f32(y[(size_t)s * p.ldy + c]) : st[(size_t)(hist + (s - first)) * C + c];
        acc += load_w(p.cw, p.cw_f32, (size_t)c * p.taps + j) * v;
        if (p.own_state && j > 0) st[(size_t)(j - 1) * C + c] = v;
      }
      crow[c] = acc;
      if (c < QW) ssq += acc * acc; else if (c < QW + KW) ssk += acc * acc;
    }
  }
  float rq = 1.f, rk = 1.f;
  if (p.qw) rq = 1.0f / sqrtf(block_sum(ssq, red) / (float)QW + p.eps);
  if (p.kw && p.G > 0) rk = 1.0f / sqrtf(block_sum(ssk, red) / (float)KW + p.eps);
  __syncthreads();
  size_t page_slot = (size_t)page * p.G * SLLM_PAGE + (pos % SLLM_PAGE);
  A* q_row = (A*)p.q_out + (size_t)t * p.ldq;
  A* kp = (A*)p.kpages;
  A* vp = (A*)p.vpages;
  int hd = p.hd, half = p.rot >> 1;
  const float2* csr = p.cs + (size_t)pos * half;
  if (VEC && (p.interleaved || !(half & 1))) {
    // a warp a head, a lane two neighbouring dims (both in the same half of the turning part, or a pair of their own,
    // or behind it) and one store for both: no division on the way
    int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int head = wid; head < p.H + p.G; head += nw) {
      int col = head * hd;
      bool is_q = head < p.H;
      const void* w = is_q ? p.qw : p.kw;
      int wc = is_q ? col : col - QW;
      float r = is_q ? rq : rk;
      A* dst = is_q ? q_row + col : kp + (page_slot + (size_t)(head - p.H) * SLLM_PAGE) * hd;
      for (int d = 2 * lane; d < hd; d += 64) {
        float2 x = *(const float2*)(crow + col + d);
        float w0 = 1.f, w1 = 1.f;
        if (w) { w0 = load_w(w, p.w_f32, wc + d); w1 = load_w(w, p.w_f32, wc + d + 1); }
        float o0 = x.x * r * w0, o1 = x.y * r * w1;
        if (d < p.rot) {
          if (p.interleaved) {
            float2 a = csr[d >> 1];
            float t0 = o0 * a.x - o1 * a.y;
            o1 = o1 * a.x + o0 * a.y;
            o0 = t0;
          } else {
            bool low = d < half;
            int pd = low ? d + half : d - half;                        // the partner dims
            float2 y = *(const float2*)(crow + col + pd);
            float v0 = 1.f, v1 = 1.f;
            if (w) { v0 = load_w(w, p.w_f32, wc + pd); v1 = load_w(w, p.w_f32, wc + pd + 1); }
            float p0 = y.x * r * v0, p1 = y.y * r * v1;
            int ci = low ? d : pd;
            float2 a = csr[ci], bb = csr[ci + 1];
            o0 = low ? o0 * a.x - p0 * a.y : o0 * a.x + p0 * a.y;
            o1 = low ? o1 * bb.x - p1 * bb.y : o1 * bb.x + p1 * bb.y;
          }
        }
        st2(dst + d, o0, o1);
      }
    }
    for (int g = wid; g < p.G; g += nw)
      for (int j = 4 * lane; j < p.vd; j += 128)
        st4(vp + (page_slot + (size_t)g * SLLM_PAGE) * p.vd + j, *(const float4*)(crow + QW + KW + g * p.vd + j));
    return;
  }
  for (int idx = threadIdx.x; idx < (p.H + p.G) * half; idx += blockDim.x) {
    int head = idx / half, i = idx % half;
    int i0 = p.interleaved ? 2 * i : i, i1 = p.interleaved ? 2 * i + 1 : i + half;
    int col = head * hd;
    bool is_q = head < p.H;
    const void* w = is_q ? p.qw : p.kw;
    int wc = is_q ? col : col - QW;
    float r = is_q ? rq : rk;
    float x0 = crow[col + i0] * r, x1 = crow[col + i1] * r;
    if (w) { x0 *= load_w(w, p.w_f32, wc + i0); x1 *= load_w(w, p.w_f32, wc + i1); }
    float2 a = csr[i];
    A* dst = is_q ? q_row + col : kp + (page_slot + (size_t)(head - p.H) * SLLM_PAGE) * hd;
    dst[i0] = from_f32<A>(x0 * a.x - x1 * a.y);
    dst[i1] = from_f32<A>(x1 * a.x + x0 * a.y);
  }
  int tail = hd - p.rot;
  for (int idx = threadIdx.x; idx < (p.H + p.G) * tail; idx += blockDim.x) {
    int head = idx / tail, j = p.rot + idx % tail;
    int col = head * hd;
    bool is_q = head < p.H;
    const void* w = is_q ? p.qw : p.kw;
    float x = crow[col + j] * (is_q ? rq : rk);
    if (w) x *= load_w(w, p.w_f32, (is_q ? col : col - QW) + j);
    A* dst = is_q ? q_row + col : kp + (page_slot + (size_t)(head - p.H) * SLLM_PAGE) * hd;
    dst[j] = from_f32<A>(x);
  }
  for (int idx = threadIdx.x; idx < p.G * p.vd; idx += blockDim.x) {
    int g = idx / p.vd, j = idx % p.vd;
    vp[(page_slot + (size_t)g * SLLM_PAGE) * p.vd + j] = from_f32<A>(crow[QW + KW + idx]);
  }
}

// After a step of several rows a sequence: the state becomes the last taps - 1 rows of [state | the step's rows].
template <typename A>
__global__ void conv_state_kernel(ConvNormArgs p, int n_seqs, int C) {
  int b = blockIdx.x;
  int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= C || b >= n_seqs) return;
  const A* y = (const A*)p.y;
  int first = p.seq_start[b], n = p.seq_start[b + 1] - first;
  int hist = p.taps - 1;
  float* st = p.state + (size_t)p.slots[b] * hist * C;
  for (int k = 0; k < hist; k++) {              // ascending: a kept entry moves down before its place is written
    int s = n + k - hist;                       // a row of the step, or (negative) an entry of the old state
    st[(size_t)k * C + c] = s >= 0 ? to_f32(y[(size_t)(first + s) * p.ldy + c]) : st[(size_t)(hist + s) * C + c];
  }
}

// ------------------------------------------------------------------ a gate per head on the attention output
// o[t][h * vd + j] *= sigmoid(g[t * ldg + h]) (g float or A), one thread per element.
template <typename A>
__global__ void head_gate_kernel(A* __restrict__ o, int ldo, const void* __restrict__ g, int g_f32, int ldg, int T, int H, int vd) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  size_t n = (size_t)T * H * vd;
  if (i >= n) return;
  int t = (int)(i / ((size_t)H * vd)), r = (int)(i % ((size_t)H * vd));
  float s = sigmoid_f(ld_flag<A>(g, g_f32, (size_t)t * ldg + r / vd));
  A* p = o + (size_t)t * ldo + r;
  *p = from_f32<A>(to_f32(*p) * s);
}

// eight neighbouring columns a thread: vd, ldo multiples of eight, o aligned for the wide access
template <typename A>
__global__ void head_gate_vec8_kernel(A* __restrict__ o, int ldo, const void* __restrict__ g, int g_f32, int ldg, int T, int H, int vd) {
  size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 8;
  size_t wrow = (size_t)H * vd;
  if (i >= (size_t)T * wrow) return;
  int t = (int)(i / wrow), r = (int)(i % wrow);
  float s = sigmoid_f(ld_flag<A>(g, g_f32, (size_t)t * ldg + r / vd));
  A* p = o + (size_t)t * ldo + r;
  F8 v = ld8(p);
#pragma unroll
  for (int k = 0; k < 8; k++) v.f[k] *= s;
  st8(p, v);
}

// four neighbouring columns a thread: vd, ldo multiples of four, o aligned for the wide access
template <typename A>
__global__ void head_gate_vec_kernel(A* __restrict__ o, int ldo, const void* __restrict__ g, int g_f32, int ldg, int T, int H, int vd) {
  size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  size_t wrow = (size_t)H * vd;
  if (i >= (size_t)T * wrow) return;
  int t = (int)(i / wrow), r = (int)(i % wrow);
  float s = sigmoid_f(ld_flag<A>(g, g_f32, (size_t)t * ldg + r / vd));
  A* p = o + (size_t)t * ldo + r;
  float4 v = ld4(p);
  st4(p, make_float4(v.x * s, v.y * s, v.z * s, v.w * s));
}

// a logit per element (vd == 1), eight neighbouring columns a thread: o[t][j] *= sigmoid(g[t][j]), g of the element type;
// n, ldo, ldg multiples of eight, both aligned for the wide access
template <typename A>
__global__ void elem_gate_vec8_kernel(A* __restrict__ o, int ldo, const A* __restrict__ g, int ldg, int T, int n) {
  size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (i >= (size_t)T * n) return;
  int t = (int)(i / n), r = (int)(i % n);
  A* p = o + (size_t)t * ldo + r;
  F8 v = ld8(p), w = ld8(g + (size_t)t * ldg + r);
#pragma unroll
  for (int k = 0; k < 8; k++) v.f[k] *= sigmoid_f(w.f[k]);
  st8(p, v);
}

// ------------------------------------------------------------------ the stream takes its pending addend; a copy in A
// x float [n] += sum over p < P of d[p * n + i] (d float or A; P == 0: nothing to add); xb[i] = A(x[i]).
template <typename A>
__global__ void add_cast_kernel(float* __restrict__ x, const void* __restrict__ d, int d_f32, int P, A* __restrict__ xb, size_t n) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  float v = x[i];
  for (int p = 0; p < P; p++) v += ld_flag<A>(d, d_f32, (size_t)p * n + i);
  if (P > 0) x[i] = v;
  xb[i] = from_f32<A>(v);
}

// four elements a thread (n a multiple of four)
template <typename A>
__global__ void add_cast_vec_kernel(float* __restrict__ x, const void* __restrict__ d, int d_f32, int P, A* __restrict__ xb, size_t n) {
  size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (i >= n) return;
  float4 v = *(const float4*)(x + i);
  for (int p = 0; p < P; p++) {
    float4 a = ld4f<A>(d, d_f32, (size_t)p * n + i);
    v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
  }
  if (P > 0) *(float4*)(x + i) = v;
  st4(xb + i, v);
}

// several addends at once: x float [T][d] += sum over the list's entries k, each [P_k][T][d] partial sums (float or A) added in
// their order, and + vec[j] (float [d], or null) on every row; xb (A, or null) = the rounded stream. One pass over the stream.
#define GATE_MAX_ADDENDS 8
struct AddList {
  const void* p[GATE_MAX_ADDENDS];
  int f32[GATE_MAX_ADDENDS];
  int P[GATE_MAX_ADDENDS];
  int count;
};
template <typename A>
__global__ void add_list_cast_kernel(float* __restrict__ x, AddList l, const float* __restrict__ vec, int d, A* __restrict__ xb, size_t n) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  float v = x[i];
  for (int k = 0; k < l.count; k++)
    for (int q = 0; q < l.P[k]; q++) v += ld_flag<A>(l.p[k], l.f32[k], (size_t)q * n + i);
  if (vec) v += vec[i % d];
  x[i] = v;
  if (xb) xb[i] = from_f32<A>(v);
}
template <typename A>
__global__ void add_list_cast_vec_kernel(float* __restrict__ x, AddList l, const float* __restrict__ vec, int d, A* __restrict__ xb, size_t n) {
  size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (i >= n) return;
  float4 v = *(const float4*)(x + i);
  for (int k = 0; k < l.count; k++)
    for (int q = 0; q < l.P[k]; q++) {
      float4 a = ld4f<A>(l.p[k], l.f32[k], (size_t)q * n + i);
      v.x += a.x; v.y += a.y; v.z += a.z; v.w += a.w;
    }
  if (vec) {
    float4 b = *(const float4*)(vec + i % d);
    v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
  }
  *(float4*)(x + i) = v;
  if (xb) st4(xb + i, v);
}

// ------------------------------------------------------------------ gelu(a) * a slice of the token's table row
// out[t][j] = gelu_tanh(a[t][j]) * table[ids[t]][col0 + j], j < D; table [rows][ldt] of A.
template <typename A>
__global__ void gelu_mul_rows_kernel(const A* __restrict__ a, int lda, const int* __restrict__ ids, const A* __restrict__ table,
                                     int ldt, int col0, A* __restrict__ out, int T, int D) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)T * D) return;
  int t = (int)(i / D), j = (int)(i % D);
  float e = to_f32(table[(size_t)ids[t] * ldt + col0 + j]);
  out[i] = from_f32<A>(gelu_tanh_f(to_f32(a[(size_t)t * lda + j])) * e);
}

// ------------------------------------------------------------------ x += (y + yb) / rms(y + yb) * w
// y float or A: [P][T][d] partial sums added in their order, then yb (float [d], the product's bias, or null); a block per
// row, the row's y kept in shared memory.
// With `out` (A, [gridDim.x][d]) the row's norm for the next reader follows in the same pass: out = x / rms(x) * w2 of
// the stream as it now stands, or with `b2` the norm without statistics tanh(alpha2 x) * w2 + b2 (w2, b2 float then);
// without w2 it is the stream's row itself in the element type. `rows` (or null) picks the stream's rows that are worked on,
// out's rows stay in order. `vec` (float [d], or null) is added to the row as well.
template <typename A>
__global__ void add_rms_normed_kernel(float* x, const void* y, int y_f32, int P, int T, const float* yb,
                                      const void* __restrict__ w, int w_f32, int d, float eps, const int* __restrict__ rows,
                                      const void* __restrict__ w2, int w2_f32, float eps2, A* out,
                                      const float* __restrict__ vec, const float* __restrict__ b2, float alpha2) {
  extern __shared__ __align__(16) float rowbuf[];
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  int t = rows ? rows[blockIdx.x] : blockIdx.x;
  float ss = 0.f;
  for (int j = threadIdx.x; j < d; j += blockDim.x) {
    float v = 0.f;
    for (int p = 0; p < P; p++) v += ld_flag<A>(y, y_f32, ((size_t)p * T + t) * d + j);
    if (yb) v += yb[j];
    rowbuf[j] = v;
    ss += v * v;
  }
  float r = 1.0f / sqrtf(block_sum(ss, red) / (float)d + eps);
  float ss2 = 0.f;
  for (int j = threadIdx.x; j < d; j += blockDim.x) {
    float v = x[(size_t)t * d + j] + rowbuf[j] * r * load_w(w, w_f32, j);
    if (vec) v += vec[j];
    x[(size_t)t * d + j] = v;
    if (out && !w2) out[(size_t)blockIdx.x * d + j] = from_f32<A>(v);
    rowbuf[j] = v;                             // a column is one thread's in every pass
    ss2 += v * v;
  }
  if (!out || !w2) return;
  if (b2) {
    for (int j = threadIdx.x; j < d; j += blockDim.x)
      out[(size_t)blockIdx.x * d + j] = from_f32<A>(tanhf(alpha2 * rowbuf[j]) * load_w(w2, 1, j) + b2[j]);
    return;
  }
  float r2 = 1.0f / sqrtf(block_sum(ss2, red) / (float)d + eps2);
  for (int j = threadIdx.x; j < d; j += blockDim.x)
    out[(size_t)blockIdx.x * d + j] = from_f32<A>(rowbuf[j] * r2 * load_w(w2, w2_f32, j));
}

// The same for rows that fit a block's registers, NV accesses of four columns a thread: the stream's row is asked for together
// with the addend, and neither passes through shared memory.
struct RmsAddArgs {
  float* x; const void* y; int y_f32, P, T; const float* yb; const void* w; int w_f32, d; float eps; const int* rows;
  const void* w2; int w2_f32; float eps2; void* out; const float* vec; const float* b2; float alpha2;
};
__device__ __forceinline__ float4 load_w4(const void* w, int is_f32, int j) {
  return is_f32 ? *(const float4*)((const float*)w + j) : ld4((const bf16*)w + j);
}
__device__ __forceinline__ float dot4(const float4& a) { return fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(a.z, a.z, a.w * a.w))); }

template <typename A, int NV>
__global__ void __launch_bounds__(NV == 4 ? 512 : 1024) add_rms_normed_reg_kernel(RmsAddArgs p) {
  __shared__ float red[2][32];
  pdl_launch_dependents();
  const int d = p.d, step = blockDim.x * 4, j0 = threadIdx.x * 4;
  float4 w[NV];
#pragma unroll
  for (int n = 0; n < NV; n++)
    if (j0 + n * step < d) w[n] = load_w4(p.w, p.w_f32, j0 + n * step);      // a weight: no kernel of the step writes it
  pdl_wait();
  const int t = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  float* xr = p.x + (size_t)t * d;
  float4 x[NV], y[NV];
#pragma unroll
  for (int n = 0; n < NV; n++) {
    const int j = j0 + n * step;
    if (j < d) {
      y[n] = ld4f<A>(p.y, p.y_f32, (size_t)t * d + j);
      x[n] = *(const float4*)(xr + j);
    }
  }
  for (int q = 1; q < p.P; q++) {
#pragma unroll
    for (int n = 0; n < NV; n++) {
      const int j = j0 + n * step;
      if (j < d) {
        const float4 a = ld4f<A>(p.y, p.y_f32, ((size_t)q * p.T + t) * d + j);
        y[n].x += a.x; y[n].y += a.y; y[n].z += a.z; y[n].w += a.w;
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int n = 0; n < NV; n++) {
    const int j = j0 + n * step;
    if (j >= d) continue;
    if (p.yb) {
      const float4 b = *(const float4*)(p.yb + j);
      y[n].x += b.x; y[n].y += b.y; y[n].z += b.z; y[n].w += b.w;
    }
    ss += dot4(y[n]);
  }
  const float r = 1.0f / sqrtf(block_sum(ss, red[0]) / (float)d + p.eps);
  A* out = (A*)p.out + (size_t)blockIdx.x * d;
  float ss2 = 0.f;
#pragma unroll
  for (int n = 0; n < NV; n++) {
    const int j = j0 + n * step;
    if (j >= d) continue;
    float4 v = x[n];
    v.x += y[n].x * r * w[n].x; v.y += y[n].y * r * w[n].y; v.z += y[n].z * r * w[n].z; v.w += y[n].w * r * w[n].w;
    if (p.vec) {
      const float4 b = *(const float4*)(p.vec + j);
      v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
    }
    *(float4*)(xr + j) = v;
    x[n] = v;
    if (p.out && !p.w2) st4(out + j, v);
    ss2 += dot4(v);
  }
  if (!p.out || !p.w2) return;
  const float r2 = p.b2 ? 0.f : 1.0f / sqrtf(block_sum(ss2, red[1]) / (float)d + p.eps2);
#pragma unroll
  for (int n = 0; n < NV; n++) {
    const int j = j0 + n * step;
    if (j >= d) continue;
    const float4 v = x[n], u = load_w4(p.w2, p.w2_f32, j);
    if (p.b2) {
      const float4 b = *(const float4*)(p.b2 + j);
      st4(out + j, make_float4(tanhf(p.alpha2 * v.x) * u.x + b.x, tanhf(p.alpha2 * v.y) * u.y + b.y, tanhf(p.alpha2 * v.z) * u.z + b.z,
                               tanhf(p.alpha2 * v.w) * u.w + b.w));
    } else {
      st4(out + j, make_float4(v.x * r2 * u.x, v.y * r2 * u.y, v.z * r2 * u.z, v.w * r2 * u.w));
    }
  }
}

// ------------------------------------------------------------------ cap * tanh(x * scale / cap) (cap <= 0: x * scale)
__global__ void softcap_kernel(float* __restrict__ x, size_t n, float cap, float scale) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  float v = x[i] * scale;
  x[i] = cap > 0.f ? cap * tanhf(v / cap) : v;
}

}  // namespace gate

// The state-space recurrence with one decay per head and token (the mixer of Mamba-2), for float and bfloat16 activations (A).
//
// Per head h (group g = h / (H / G)) a state S [N, V]: with dt_t = softplus(raw_t + bias_h) and a_t = -exp(A_log_h) dt_t,
//   S_t = exp(a_t) S_{t-1} + dt_t B_t x_t^T;   y_t = S_t^T C_t + D_h x_t;   out_t = y_t silu(z_t).
// Columns of a row of xbc: [x: H V | B: G N | C: G N] (element type). The state [slot][H][N][V] is float, read at a step's start
// and left at its end. Step sizes, decays, exponentials, state and sums are float; out is of the element type.
//
//   ssd_walk           token by token with the state in registers: decode steps, short runs, and all of 32-bit
//   ssd_chunk_states   bfloat16, long runs: what every chunk of SSD_Q rows adds to the state
//   ssd_chunk_pass     the state in front of every chunk, and the state left at the end
//   ssd_chunk_scan     every chunk's output from the state in front of it and its own rows
//   group_norm         equal runs of columns over their own root mean square, times a weight
//
// With `w` the out rows are multiplied by a weight per column, and with `sumsq` every (row, block of columns) leaves the sum
// of squares of y silu(z) in front of that weight: the halves of an RMS norm over the whole row that the product behind it
// can finish.
#pragma once
#include "common.cuh"

namespace ssd {

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

struct Args {
  const void* xbc; int ldx;
  const void* dt; int lddt;              // raw step sizes [T, H] (element type, a column slice)
  const float* dt_bias; const float* a_log; const float* dskip;   // [H]
  const void* z; int ldz;                // [T, H V]
  float* state;                          // [slots][H][N][V]
  const int* seq_start; const int* slots;
  void* out; int ldo;                    // [T, H V]
  const float* w;                        // [H V] or null
  float* sumsq;                          // [H * column blocks][T] or null
  int T, H, G, V, N;
  float* chunk_state;                    // chunked form: [chunks][H][N][V]
  float* chunk_decay;                    // [chunks][H]
  int vec;                               // rows of xbc, their parts and V allow 16-byte accesses
};

// ------------------------------------------------------------------ token by token
// A block of 8 warps takes 32 columns of one head of one sequence. Lane (vl, nl) = (lane & 7, lane >> 3) of warp w holds the
// columns 4 vl .. 4 vl + 3 of the state rows n = 32 i + 4 w + nl, i < NPT. Rows come in tiles of up to R: a row's partial
// read-outs are folded over the warp's four rows of lanes, the warps' parts meet in shared memory once a tile.
template <typename A, int NPT>
__global__ void __launch_bounds__(256) ssd_walk_kernel(Args p, int R) {
  extern __shared__ __align__(16) float sm[];
  const int N = p.N, V = p.V;
  float* red = sm;                       // [R][8][32]; what is read four floats at a time comes first, whatever R and N are
  float* x_s = red + R * 256;            // [R][32]
  float* b_s = x_s + R * 32;             // [R][N]
  float* c_s = b_s + R * N;              // [R][N]
  float* dt_s = c_s + R * N;             // [R]
  float* dec_s = dt_s + R;               // [R]
  const int vblocks = (V + 31) / 32;
  const int h = blockIdx.x / vblocks, v0 = (blockIdx.x % vblocks) * 32, b = blockIdx.y;
  const int g = h / (p.H / p.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, vl = lane & 7, nl = lane >> 3;
  const int r_begin = p.seq_start[b], r_end = p.seq_start[b + 1];
  const int HV = p.H * V;
  const A* xbc = (const A*)p.xbc;
  const A* dtr = (const A*)p.dt;
  const A* zr = (const A*)p.z;
  const float a = -expf(p.a_log[h]), bias = p.dt_bias[h], dsk = p.dskip[h];
  float* st = p.state + ((size_t)p.slots[b] * p.H + h) * N * V;
  const int vc = v0 + 4 * vl;
  const bool whole = (V & 3) == 0;       // a lane's four columns: all there or none

  float S[NPT][4];
#pragma unroll
  for (int i = 0; i < NPT; i++) {
    const int n = 32 * i + 4 * warp + nl;
    S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
    if (n < N) {
      if (whole) {
        if (vc < V) {
          float4 q = *(const float4*)(st + (size_t)n * V + vc);
          S[i][0] = q.x; S[i][1] = q.y; S[i][2] = q.z; S[i][3] = q.w;
        }
      } else {
#pragma unroll
        for (int e = 0; e < 4; e++)
          if (vc + e < V) S[i][e] = st[(size_t)n * V + vc + e];
      }
    }
  }
  for (int r0 = r_begin; r0 < r_end; r0 += R) {
    const int n_rows = min(R, r_end - r0);
    __syncthreads();
    for (int i = threadIdx.x; i < n_rows * N; i += 256) {
      const int r = i / N, n = i % N;
      const A* row = xbc + (size_t)(r0 + r) * p.ldx + HV + (size_t)g * N + n;
      b_s[i] = to_f32(row[0]);
      c_s[i] = to_f32(row[(size_t)p.G * N]);
    }
    for (int i = threadIdx.x; i < n_rows * 32; i += 256) {
      const int r = i >> 5, v = v0 + (i & 31);
      x_s[i] = v < V ? to_f32(xbc[(size_t)(r0 + r) * p.ldx + (size_t)h * V + v]) : 0.f;
    }
    for (int r = threadIdx.x; r < n_rows; r += 256) {
      const float d = softplus_f(to_f32(dtr[(size_t)(r0 + r) * p.lddt + h]) + bias);
      dt_s[r] = d;
      dec_s[r] = expf(a * d);
    }
    __syncthreads();
    for (int r = 0; r < n_rows; r++) {
      const float dec = dec_s[r], d = dt_s[r];
      const float4 x = *(const float4*)(x_s + r * 32 + 4 * vl);
      const float dx0 = d * x.x, dx1 = d * x.y, dx2 = d * x.z, dx3 = d * x.w;
      float y0 = 0.f, y1 = 0.f, y2 = 0.f, y3 = 0.f;
#pragma unroll
      for (int i = 0; i < NPT; i++) {
        const int n = 32 * i + 4 * warp + nl;
        if (n < N) {
          const float bn = b_s[r * N + n], cn = c_s[r * N + n];
          S[i][0] = fmaf(dec, S[i][0], bn * dx0); y0 = fmaf(cn, S[i][0], y0);
          S[i][1] = fmaf(dec, S[i][1], bn * dx1); y1 = fmaf(cn, S[i][1], y1);
          S[i][2] = fmaf(dec, S[i][2], bn * dx2); y2 = fmaf(cn, S[i][2], y2);
          S[i][3] = fmaf(dec, S[i][3], bn * dx3); y3 = fmaf(cn, S[i][3], y3);
        }
      }
#pragma unroll
      for (int o = 8; o <= 16; o <<= 1) {
        y0 += __shfl_xor_sync(0xffffffffu, y0, o);
        y1 += __shfl_xor_sync(0xffffffffu, y1, o);
        y2 += __shfl_xor_sync(0xffffffffu, y2, o);
        y3 += __shfl_xor_sync(0xffffffffu, y3, o);
      }
      if (nl == 0) *(float4*)(red + (r * 8 + warp) * 32 + 4 * vl) = make_float4(y0, y1, y2, y3);
    }
    __syncthreads();
    for (int r = warp; r < n_rows; r += 8) {       // a warp a row, a lane a column
      const int v = v0 + lane;
      float y = 0.f;
#pragma unroll
      for (int w = 0; w < 8; w++) y += red[(r * 8 + w) * 32 + lane];
      float u = 0.f;
      if (v < V) {
        const size_t col = (size_t)h * V + v;
        u = fmaf(dsk, x_s[r * 32 + lane], y) * silu_f(to_f32(zr[(size_t)(r0 + r) * p.ldz + col]));
        ((A*)p.out)[(size_t)(r0 + r) * p.ldo + col] = from_f32<A>(p.w ? u * p.w[col] : u);
      }
      if (p.sumsq) {
        const float q = warp_sum(u * u);
        if (lane == 0) p.sumsq[(size_t)blockIdx.x * p.T + r0 + r] = q;
      }
    }
  }
  if (r_end > r_begin) {
#pragma unroll
    for (int i = 0; i < NPT; i++) {
      const int n = 32 * i + 4 * warp + nl;
      if (n < N) {
        if (whole) {
          if (vc < V) *(float4*)(st + (size_t)n * V + vc) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
        } else {
#pragma unroll
          for (int e = 0; e < 4; e++)
            if (vc + e < V) st[(size_t)n * V + vc + e] = S[i][e];
        }
      }
    }
  }
}

// ------------------------------------------------------------------ in chunks, on the tensor cores
// A sequence's rows are cut into chunks of SSD_Q. With c_i the sum of a over the chunk's rows up to and with i:
//   y_i = exp(c_i) S^T C_i + sum_{j <= i} exp(c_i - c_j) dt_j (C_i . B_j) x_j + D x_i          (S in front of the chunk)
//   S  <- exp(c_last) S + sum_j exp(c_last - c_j) dt_j B_j x_j^T.
// x, B and C are bfloat16 as they come, so C . B is exact in a bfloat16 product with float sums. What is float (the state, and
// everything that carries a step size or a decay) enters a product as the sum of three bfloat16 numbers (split3): 24 bits of
// mantissa, so nothing is lost against float. c is summed in double and kept as two floats, so that differences of sums that
// have grown large keep their digits.
#define SSD_Q 128
#define SSD_VB 64            // value columns a block
#define SSD_VS (SSD_VB + 8)  // padded row of a tile of them (elements)

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const bf16* p) {
  uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const bf16* p) {
  uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a) : "memory");
}
__device__ __forceinline__ void split3(float v, bf16& a, bf16& b, bf16& c) {
  a = __float2bfloat16_rn(v);
  const float r = v - __bfloat162float(a);
  b = __float2bfloat16_rn(r);
  c = __float2bfloat16_rn(r - __bfloat162float(b));
}
__device__ __forceinline__ uint32_t pack2(bf16 a, bf16 b) {
  __nv_bfloat162 v;
  v.x = a; v.y = b;
  return *(uint32_t*)&v;
}
// two neighbouring floats as three packed pairs
__device__ __forceinline__ void split3_pair(float u, float v, uint32_t& p0, uint32_t& p1, uint32_t& p2) {
  bf16 a0, b0, c0, a1, b1, c1;
  split3(u, a0, b0, c0);
  split3(v, a1, b1, c1);
  p0 = pack2(a0, a1); p1 = pack2(b0, b1); p2 = pack2(c0, c1);
}

// rows [0, SSD_Q) of `cols` columns (row stride ldx) into a tile of row stride `s`; rows from n on and columns from `cols` up
// to `cols_p` (a multiple of 8) are zero
__device__ __forceinline__ void stage_rows(bf16* dst, int s, const bf16* src, int ldx, int n, int cols, int cols_p, int vec) {
  if (vec) {
    const int ch = cols_p >> 3;
    for (int i = threadIdx.x; i < SSD_Q * ch; i += 256) {
      const int r = i / ch, c = (i % ch) << 3;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < n && c < cols) v = *(const uint4*)(src + (size_t)r * ldx + c);
      *(uint4*)(dst + r * s + c) = v;
    }
  } else {
    for (int i = threadIdx.x; i < SSD_Q * cols_p; i += 256) {
      const int r = i / cols_p, c = i % cols_p;
      dst[r * s + c] = r < n && c < cols ? src[(size_t)r * ldx + c] : __float2bfloat16_rn(0.f);
    }
  }
}

// step sizes of the chunk's rows and the running sums of a, the first warp's work (rows from n on: dt 0)
__device__ __forceinline__ void chunk_sums(const Args& p, int row, int n, int h, float* dt_s, float* hi, float* lo) {
  if (threadIdx.x >= 32) return;
  constexpr int PER = SSD_Q / 32;
  const int lane = threadIdx.x;
  const double a = -(double)expf(p.a_log[h]);
  const float bias = p.dt_bias[h];
  float d[PER];
  double c[PER], sum = 0.0;
#pragma unroll
  for (int k = 0; k < PER; k++) {
    const int r = lane * PER + k;
    d[k] = r < n ? softplus_f(to_f32(((const bf16*)p.dt)[(size_t)(row + r) * p.lddt + h]) + bias) : 0.f;
    sum += a * (double)d[k];
    c[k] = sum;
  }
  double before = sum;                   // inclusive over the lanes, then made exclusive
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double u = __shfl_up_sync(0xffffffffu, before, o);
    if (lane >= o) before += u;
  }
  before -= sum;
#pragma unroll
  for (int k = 0; k < PER; k++) {
    const double t = before + c[k];
    dt_s[lane * PER + k] = d[k];
    hi[lane * PER + k] = (float)t;
    lo[lane * PER + k] = (float)(t - (double)(float)t);
  }
}

// A sequence's chunks lie one behind the other from this one on: the ranges of two sequences never meet, because
// ceil(len / Q) <= floor((start + len) / Q) - floor(start / Q) + 1. There are at most T / Q + sequences of them.
__device__ __forceinline__ size_t first_chunk(int start, int b) { return (size_t)(start / SSD_Q + b); }

// U = sum_j B_j (w_j x_j)^T, w_j = exp(c_last - c_j) dt_j. A warp takes 16 state rows at a time (M) against the block's 64
// columns; the contraction runs over the chunk's rows: both operands are read transposed from row-major tiles.
__global__ void __launch_bounds__(256) ssd_chunk_states_kernel(Args p) {
  extern __shared__ __align__(16) bf16 smb[];
  __shared__ float dt_s[SSD_Q], hi[SSD_Q], lo[SSD_Q];
  const int b = blockIdx.z, start = p.seq_start[b], len = p.seq_start[b + 1] - start;
  const int r0 = blockIdx.x * SSD_Q;
  if (r0 >= len) return;
  const int n = min(SSD_Q, len - r0), row = start + r0;
  const int vblocks = (p.V + SSD_VB - 1) / SSD_VB;
  const int h = blockIdx.y / vblocks, v0 = (blockIdx.y % vblocks) * SSD_VB, g = h / (p.H / p.G);
  const int Np = (p.N + 15) & ~15, NS = Np + 8, vn = min(SSD_VB, p.V - v0);
  bf16* Bs = smb;                        // [Q][NS]
  bf16* Xs = Bs + SSD_Q * NS;            // 3 x [Q][VS]
  const bf16* xbc = (const bf16*)p.xbc + (size_t)row * p.ldx;
  chunk_sums(p, row, n, h, dt_s, hi, lo);
  stage_rows(Bs, NS, xbc + (size_t)p.H * p.V + (size_t)g * p.N, p.ldx, n, p.N, Np, p.vec);
  __syncthreads();
  const float last_hi = hi[SSD_Q - 1], last_lo = lo[SSD_Q - 1];     // rows past n add nothing to the sum
  const bf16* xr = xbc + (size_t)h * p.V + v0;
  for (int i = threadIdx.x; i < SSD_Q * (SSD_VB / 2); i += 256) {
    const int r = i / (SSD_VB / 2), c = (i % (SSD_VB / 2)) * 2;
    float u = 0.f, v = 0.f;
    if (r < n && c < vn) {
      const float w = expf((last_hi - hi[r]) + (last_lo - lo[r])) * dt_s[r];
      if (p.vec) {
        const __nv_bfloat162 q = *(const __nv_bfloat162*)(xr + (size_t)r * p.ldx + c);
        u = w * __low2float(q); v = w * __high2float(q);
      } else {
        u = w * to_f32(xr[(size_t)r * p.ldx + c]);
        v = c + 1 < vn ? w * to_f32(xr[(size_t)r * p.ldx + c + 1]) : 0.f;
      }
    }
    uint32_t q0, q1, q2;
    split3_pair(u, v, q0, q1, q2);
    *(uint32_t*)(Xs + r * SSD_VS + c) = q0;
    *(uint32_t*)(Xs + (SSD_Q + r) * SSD_VS + c) = q1;
    *(uint32_t*)(Xs + (2 * SSD_Q + r) * SSD_VS + c) = q2;
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t chunk = first_chunk(start, b) + blockIdx.x;
  float* dst = p.chunk_state + (chunk * p.H + h) * (size_t)p.N * p.V;
  if (v0 == 0 && threadIdx.x == 0) p.chunk_decay[chunk * p.H + h] = expf(last_hi + last_lo);
  const int ksteps = (n + 15) / 16;
  for (int mt = warp; mt < Np / 16; mt += 8) {
    float acc[SSD_VB / 8][4];
#pragma unroll
    for (int i = 0; i < SSD_VB / 8; i++) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int ks = 0; ks < ksteps; ks++) {
      uint32_t a[4];
      ldsm4t(a, Bs + (ks * 16 + (lane & 7) + (lane >> 4) * 8) * NS + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int part = 0; part < 3; part++) {
        const bf16* xt = Xs + (part * SSD_Q + ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SSD_VS + (lane >> 4) * 8;
#pragma unroll
        for (int nt = 0; nt < SSD_VB / 16; nt++) {
          uint32_t q[4];
          ldsm4t(q, xt + nt * 16);
          mma_bf16(acc[2 * nt], a, q[0], q[1]);
          mma_bf16(acc[2 * nt + 1], a, q[2], q[3]);
        }
      }
    }
    const int ra = mt * 16 + (lane >> 2), rb = ra + 8;
#pragma unroll
    for (int i = 0; i < SSD_VB / 8; i++) {
      const int c = i * 8 + (lane & 3) * 2;
      if (c < vn) {
        if (ra < p.N) dst[(size_t)ra * p.V + v0 + c] = acc[i][0];
        if (rb < p.N) dst[(size_t)rb * p.V + v0 + c] = acc[i][2];
      }
      if (c + 1 < vn) {
        if (ra < p.N) dst[(size_t)ra * p.V + v0 + c + 1] = acc[i][1];
        if (rb < p.N) dst[(size_t)rb * p.V + v0 + c + 1] = acc[i][3];
      }
    }
  }
}

// Per element of a head's state, over the chunks in order: what a chunk adds is replaced by the state in front of it. E
// elements a thread (4 where they come in fours).
template <int E>
__global__ void __launch_bounds__(256) ssd_chunk_pass_kernel(Args p) {
  const int b = blockIdx.z, h = blockIdx.y, start = p.seq_start[b], len = p.seq_start[b + 1] - start;
  const int NV = p.N * p.V, e0 = (blockIdx.x * 256 + threadIdx.x) * E;
  if (e0 >= NV || len <= 0) return;
  const int chunks = (len + SSD_Q - 1) / SSD_Q;
  const size_t first = first_chunk(start, b), stride = (size_t)p.H * NV;
  float* u = p.chunk_state + (first * p.H + h) * (size_t)NV + e0;
  const float* dec = p.chunk_decay + first * p.H + h;
  float* st = p.state + ((size_t)p.slots[b] * p.H + h) * NV + e0;
  float s[E];
#pragma unroll
  for (int e = 0; e < E; e++) s[e] = st[e];
  constexpr int AHEAD = 4;
  for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
    float add[AHEAD][E], d[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; k++)
      if (c0 + k < chunks) {
        d[k] = dec[(size_t)(c0 + k) * p.H];
        if constexpr (E == 4) {
          const float4 q = *(const float4*)(u + (c0 + k) * stride);
          add[k][0] = q.x; add[k][1] = q.y; add[k][2] = q.z; add[k][3] = q.w;
        } else {
#pragma unroll
          for (int e = 0; e < E; e++) add[k][e] = u[(c0 + k) * stride + e];
        }
      }
#pragma unroll
    for (int k = 0; k < AHEAD; k++)
      if (c0 + k < chunks) {
        if constexpr (E == 4) *(float4*)(u + (c0 + k) * stride) = make_float4(s[0], s[1], s[2], s[3]);
        else {
#pragma unroll
          for (int e = 0; e < E; e++) u[(c0 + k) * stride + e] = s[e];
        }
#pragma unroll
        for (int e = 0; e < E; e++) s[e] = fmaf(d[k], s[e], add[k][e]);
      }
  }
#pragma unroll
  for (int e = 0; e < E; e++) st[e] = s[e];
}

// A chunk's output. A warp takes 16 of the chunk's rows (M). First C_i against the state in front of the chunk, times
// exp(c_i); then, 16 earlier rows j at a time, the products C_i . B_j become weights in registers (the accumulators of one
// product are the other's A operand as they stand) that meet x_j. The state's tile and the tiles of B and x share their place.
__global__ void __launch_bounds__(256) ssd_chunk_scan_kernel(Args p) {
  extern __shared__ __align__(16) bf16 smb[];
  __shared__ float dt_s[SSD_Q], hi[SSD_Q], lo[SSD_Q];
  const int b = blockIdx.z, start = p.seq_start[b], len = p.seq_start[b + 1] - start;
  const int r0 = blockIdx.x * SSD_Q;
  if (r0 >= len) return;
  const int n = min(SSD_Q, len - r0), row = start + r0;
  const int vblocks = (p.V + SSD_VB - 1) / SSD_VB;
  const int h = blockIdx.y / vblocks, v0 = (blockIdx.y % vblocks) * SSD_VB, g = h / (p.H / p.G);
  const int Np = (p.N + 15) & ~15, NS = Np + 8, vn = min(SSD_VB, p.V - v0);
  bf16* Cs = smb;                        // [Q][NS]
  bf16* Ss = Cs + SSD_Q * NS;            // 3 x [Np][VS], later
  bf16* Bs = Ss;                         // [Q][NS]
  bf16* Xs = Bs + SSD_Q * NS;            // [Q][VS]
  const bf16* xbc = (const bf16*)p.xbc + (size_t)row * p.ldx;
  const bf16* bsrc = xbc + (size_t)p.H * p.V + (size_t)g * p.N;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, t = lane & 3;
  const size_t chunk = first_chunk(start, b) + blockIdx.x;
  chunk_sums(p, row, n, h, dt_s, hi, lo);
  stage_rows(Cs, NS, bsrc + (size_t)p.G * p.N, p.ldx, n, p.N, Np, p.vec);
  {
    const float* st = p.chunk_state + (chunk * p.H + h) * (size_t)p.N * p.V + v0;
    for (int i = threadIdx.x; i < Np * (SSD_VB / 2); i += 256) {
      const int r = i / (SSD_VB / 2), c = (i % (SSD_VB / 2)) * 2;
      float u = 0.f, v = 0.f;
      if (r < p.N && c < vn) {
        if (p.vec) {
          const float2 q = *(const float2*)(st + (size_t)r * p.V + c);
          u = q.x; v = q.y;
        } else {
          u = st[(size_t)r * p.V + c];
          v = c + 1 < vn ? st[(size_t)r * p.V + c + 1] : 0.f;
        }
      }
      uint32_t q0, q1, q2;
      split3_pair(u, v, q0, q1, q2);
      *(uint32_t*)(Ss + r * SSD_VS + c) = q0;
      *(uint32_t*)(Ss + (Np + r) * SSD_VS + c) = q1;
      *(uint32_t*)(Ss + (2 * Np + r) * SSD_VS + c) = q2;
    }
  }
  __syncthreads();
  float acc[SSD_VB / 8][4];
#pragma unroll
  for (int i = 0; i < SSD_VB / 8; i++) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  const bool work = warp * 16 < n;
  const bf16* crow = Cs + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * NS + (lane >> 4) * 8;
  const int ia = warp * 16 + gr, ib = ia + 8;
  const float hia = hi[ia], loa = lo[ia], hib = hi[ib], lob = lo[ib];
  if (work) {
    for (int ks = 0; ks < Np / 16; ks++) {
      uint32_t a[4];
      ldsm4(a, crow + ks * 16);
#pragma unroll
      for (int part = 0; part < 3; part++) {
        const bf16* s = Ss + (part * Np + ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SSD_VS + (lane >> 4) * 8;
#pragma unroll
        for (int nt = 0; nt < SSD_VB / 16; nt++) {
          uint32_t q[4];
          ldsm4t(q, s + nt * 16);
          mma_bf16(acc[2 * nt], a, q[0], q[1]);
          mma_bf16(acc[2 * nt + 1], a, q[2], q[3]);
        }
      }
    }
    const float ea = expf(hia + loa), eb = expf(hib + lob);
#pragma unroll
    for (int i = 0; i < SSD_VB / 8; i++) { acc[i][0] *= ea; acc[i][1] *= ea; acc[i][2] *= eb; acc[i][3] *= eb; }
  }
  __syncthreads();                       // the state's tile has been read
  stage_rows(Bs, NS, bsrc, p.ldx, n, p.N, Np, p.vec);
  stage_rows(Xs, SSD_VS, xbc + (size_t)h * p.V + v0, p.ldx, n, vn, SSD_VB, p.vec);
  __syncthreads();
  if (work) {
    for (int jt = 0; jt <= warp; jt++) {
      float gm[2][4];
#pragma unroll
      for (int i = 0; i < 2; i++) gm[i][0] = gm[i][1] = gm[i][2] = gm[i][3] = 0.f;
      const bf16* brow = Bs + (jt * 16 + (lane & 7) + (lane >> 4) * 8) * NS + ((lane >> 3) & 1) * 8;
#pragma unroll 4
      for (int ks = 0; ks < Np / 16; ks++) {
        uint32_t a[4], q[4];
        ldsm4(a, crow + ks * 16);
        ldsm4(q, brow + ks * 16);
        mma_bf16(gm[0], a, q[0], q[1]);
        mma_bf16(gm[1], a, q[2], q[3]);
      }
      uint32_t w[3][4];                  // the weights as A operands: halves of 8 rows j, three parts
#pragma unroll
      for (int half = 0; half < 2; half++) {
        const int j = jt * 16 + half * 8 + 2 * t;
        const float h0 = hi[j], l0 = lo[j], d0 = dt_s[j], h1 = hi[j + 1], l1 = lo[j + 1], d1 = dt_s[j + 1];
        const float wa0 = j <= ia ? gm[half][0] * expf((hia - h0) + (loa - l0)) * d0 : 0.f;
        const float wa1 = j + 1 <= ia ? gm[half][1] * expf((hia - h1) + (loa - l1)) * d1 : 0.f;
        const float wb0 = j <= ib ? gm[half][2] * expf((hib - h0) + (lob - l0)) * d0 : 0.f;
        const float wb1 = j + 1 <= ib ? gm[half][3] * expf((hib - h1) + (lob - l1)) * d1 : 0.f;
        split3_pair(wa0, wa1, w[0][2 * half], w[1][2 * half], w[2][2 * half]);
        split3_pair(wb0, wb1, w[0][2 * half + 1], w[1][2 * half + 1], w[2][2 * half + 1]);
      }
      const bf16* xt = Xs + (jt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SSD_VS + (lane >> 4) * 8;
#pragma unroll
      for (int nt = 0; nt < SSD_VB / 16; nt++) {
        uint32_t q[4];
        ldsm4t(q, xt + nt * 16);
#pragma unroll
        for (int part = 0; part < 3; part++) {
          mma_bf16(acc[2 * nt], w[part], q[0], q[1]);
          mma_bf16(acc[2 * nt + 1], w[part], q[2], q[3]);
        }
      }
    }
  }
  if (!work) return;
  const float dsk = p.dskip[h];
  float ssa = 0.f, ssb = 0.f;
#pragma unroll
  for (int i = 0; i < SSD_VB / 8; i++) {
    const int c = i * 8 + 2 * t;
    if (c >= vn) continue;
    const size_t col = (size_t)h * p.V + v0 + c;
    const bool two = c + 1 < vn;
    const float w0 = p.w ? p.w[col] : 1.f, w1 = p.w && two ? p.w[col + 1] : 1.f;
#pragma unroll
    for (int s = 0; s < 2; s++) {
      const int r = s ? ib : ia;
      if (r >= n) continue;
      const bf16* z = (const bf16*)p.z + (size_t)(row + r) * p.ldz + col;
      bf16* o = (bf16*)p.out + (size_t)(row + r) * p.ldo + col;
      const bf16* x = Xs + r * SSD_VS + c;
      float z0, z1 = 0.f;
      if (p.vec) {
        const __nv_bfloat162 q = *(const __nv_bfloat162*)z;
        z0 = __low2float(q); z1 = __high2float(q);
      } else {
        z0 = to_f32(z[0]);
        if (two) z1 = to_f32(z[1]);
      }
      const float u0 = fmaf(dsk, to_f32(x[0]), acc[i][2 * s]) * silu_f(z0);
      const float u1 = two ? fmaf(dsk, to_f32(x[1]), acc[i][2 * s + 1]) * silu_f(z1) : 0.f;
      if (s) ssb += u0 * u0 + u1 * u1; else ssa += u0 * u0 + u1 * u1;
      if (p.vec) *(uint32_t*)o = pack2(__float2bfloat16_rn(u0 * w0), __float2bfloat16_rn(u1 * w1));
      else {
        o[0] = __float2bfloat16_rn(u0 * w0);
        if (two) o[1] = __float2bfloat16_rn(u1 * w1);
      }
    }
  }
  if (p.sumsq) {
#pragma unroll
    for (int o = 1; o <= 2; o <<= 1) {
      ssa += __shfl_xor_sync(0xffffffffu, ssa, o);
      ssb += __shfl_xor_sync(0xffffffffu, ssb, o);
    }
    if (t == 0) {
      float* q = p.sumsq + (size_t)blockIdx.y * p.T + row;
      if (ia < n) q[ia] = ssa;
      if (ib < n) q[ib] = ssb;
    }
  }
}

// ------------------------------------------------------------------ norm over equal runs of columns
// y[t][c] = u[t][c] / sqrt(mean of u[t]^2 over the run c lies in + eps) * w[c]; `groups` runs of W / groups columns, in place if
// y == u. One block a row; a run is a warp's work, or with few runs the block's.
template <typename A>
__global__ void __launch_bounds__(256) group_norm_kernel(const A* u, const float* __restrict__ w, A* y, int W, int groups, float eps) {
  __shared__ float red[32];
  pdl_launch_dependents();
  pdl_wait();
  const int run = W / groups;
  const A* src = u + (size_t)blockIdx.x * W;
  A* dst = y + (size_t)blockIdx.x * W;
  if (groups >= 8) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int g = warp; g < groups; g += blockDim.x >> 5) {
      float ss = 0.f;
      for (int j = lane; j < run; j += 32) {
        const float v = to_f32(src[g * run + j]);
        ss = fmaf(v, v, ss);
      }
      const float r = 1.0f / sqrtf(warp_sum(ss) / (float)run + eps);
      for (int j = lane; j < run; j += 32) dst[g * run + j] = from_f32<A>(to_f32(src[g * run + j]) * r * w[g * run + j]);
    }
    return;
  }
  const bool vec = (run & 3) == 0 && (((uintptr_t)u | (uintptr_t)y | (uintptr_t)w) & 15) == 0;
  for (int g = 0; g < groups; g++) {
    const A* s = src + g * run;
    float ss = 0.f;
    if (vec) {
      for (int j = threadIdx.x * 4; j < run; j += blockDim.x * 4) {
        const float4 v = ld4(s + j);
        ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
      }
    } else {
      for (int j = threadIdx.x; j < run; j += blockDim.x) {
        const float v = to_f32(s[j]);
        ss = fmaf(v, v, ss);
      }
    }
    const float r = 1.0f / sqrtf(block_sum(ss, red) / (float)run + eps);
    if (vec) {
      for (int j = threadIdx.x * 4; j < run; j += blockDim.x * 4) {
        const float4 v = ld4(s + j), q = *(const float4*)(w + g * run + j);
        st4(dst + g * run + j, make_float4(v.x * r * q.x, v.y * r * q.y, v.z * r * q.z, v.w * r * q.w));
      }
    } else {
      for (int j = threadIdx.x; j < run; j += blockDim.x) dst[g * run + j] = from_f32<A>(to_f32(s[j]) * r * w[g * run + j]);
    }
  }
}

}  // namespace ssd

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
  float* chunk_sums;                     // [chunks][H][3][SSD_Q]: step sizes; sums of a (base 2) of the chunk's rows as hi + lo
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
// mantissa, so nothing is lost against float. c is summed in double (times log2 e: the exponentials are of base 2) and kept as two
// floats, so that differences of sums that have grown large keep their digits.
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
// two neighbouring floats as three packed pairs of bfloat16 that add up to them
__device__ __forceinline__ uint32_t bits(const __nv_bfloat162& v) { return *(const uint32_t*)&v; }
__device__ __forceinline__ void split3_pair(float u, float v, uint32_t& p0, uint32_t& p1, uint32_t& p2) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(u, v);
  u -= __low2float(a); v -= __high2float(a);
  const __nv_bfloat162 b = __floats2bfloat162_rn(u, v);
  u -= __low2float(b); v -= __high2float(b);
  p0 = bits(a); p1 = bits(b); p2 = bits(__floats2bfloat162_rn(u, v));
}
// silu on its way into a bfloat16 number
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// 16 bytes into shared memory without a register, or zeros
__device__ __forceinline__ void cp16(bf16* dst, const bf16* src, bool there) {
  const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(there ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_wait() {
  asm volatile("cp.async.commit_group;" ::: "memory");
  asm volatile("cp.async.wait_group 0;" ::: "memory");
}

// rows [0, SSD_Q) of `cols` columns (row stride ldx) into a tile of COLS columns and row stride COLS + 8; rows from n on and
// columns from `cols` on are zero. cp_wait() and a barrier stand between this and a reader.
template <int COLS>
__device__ __forceinline__ void stage_rows(bf16* dst, const bf16* src, int ldx, int n, int cols, int vec) {
  if (vec) {
    constexpr int CH = COLS / 8;
#pragma unroll
    for (int i0 = 0; i0 < SSD_Q * CH; i0 += 256) {
      const int i = i0 + threadIdx.x, r = i / CH, c = (i % CH) * 8;
      const bool there = r < n && c < cols;
      cp16(dst + r * (COLS + 8) + c, there ? src + (size_t)r * ldx + c : src, there);
    }
  } else {
    for (int i = threadIdx.x; i < SSD_Q * COLS; i += 256) {
      const int r = i / COLS, c = i % COLS;
      dst[r * (COLS + 8) + c] = r < n && c < cols ? src[(size_t)r * ldx + c] : __float2bfloat16_rn(0.f);
    }
  }
}

// A sequence's chunks lie one behind the other from this one on: the ranges of two sequences never meet, because
// ceil(len / Q) <= floor((start + len) / Q) - floor(start / Q) + 1. There are at most T / Q + sequences of them.
__device__ __forceinline__ size_t first_chunk(int start, int b) { return (size_t)(start / SSD_Q + b); }

// U = sum_j B_j (w_j x_j)^T, w_j = exp(c_last - c_j) dt_j. A warp takes 16 state rows at a time (M) against the block's 64
// columns; the contraction runs over the chunk's rows: both operands are read transposed from row-major tiles. The blocks of a
// head's first columns also leave the chunk's step sizes and sums (base 2, as hi + lo) and its whole decay. NP: the state
// rows rounded up to what the kernel is built for.
template <int NP>
__global__ void __launch_bounds__(256, 2) ssd_chunk_states_kernel(Args p) {
  extern __shared__ __align__(16) bf16 smb[];
  __shared__ float w_s[SSD_Q];
  __shared__ double part_s[SSD_Q / 32];
  constexpr int NS = NP + 8;
  const int b = blockIdx.z, start = p.seq_start[b], len = p.seq_start[b + 1] - start;
  const int r0 = blockIdx.x * SSD_Q;
  if (r0 >= len) return;
  const int n = min(SSD_Q, len - r0), row = start + r0, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int vblocks = (p.V + SSD_VB - 1) / SSD_VB;
  const int h = blockIdx.y / vblocks, v0 = (blockIdx.y % vblocks) * SSD_VB, g = h / (p.H / p.G), vn = min(SSD_VB, p.V - v0);
  bf16* Bs = smb;                        // [Q][NS]
  bf16* Xs = Bs + SSD_Q * NS;            // 3 x [Q][VS]
  const bf16* xbc = (const bf16*)p.xbc + (size_t)row * p.ldx;
  const bf16* xr = xbc + (size_t)h * p.V + v0;
  const size_t chunk = first_chunk(start, b) + blockIdx.x;
  float raw = 0.f;
  if (tid < n) raw = to_f32(((const bf16*)p.dt)[(size_t)(row + tid) * p.lddt + h]);
  stage_rows<NP>(Bs, xbc + (size_t)p.H * p.V + (size_t)g * p.N, p.ldx, n, p.N, p.vec);
  constexpr int XI = SSD_Q * (SSD_VB / 8) / 256;          // eight columns of a row at a time
  uint4 xv[XI];
  if (p.vec) {
#pragma unroll
    for (int k = 0; k < XI; k++) {
      const int i = k * 256 + tid, r = i / (SSD_VB / 8), c = (i % (SSD_VB / 8)) * 8;
      xv[k] = r < n && c < vn ? *(const uint4*)(xr + (size_t)r * p.ldx + c) : make_uint4(0, 0, 0, 0);
    }
  }
  // a thread a row: its step size and the running sum of a, in double
  double c = 0.0;
  float d = 0.f;
  if (tid < SSD_Q) {
    if (tid < n) d = softplus_f(raw + p.dt_bias[h]);
    c = -(double)expf(p.a_log[h]) * 1.4426950408889634 * (double)d;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double u = __shfl_up_sync(0xffffffffu, c, o);
      if (lane >= o) c += u;
    }
    if (lane == 31) part_s[warp] = c;
  }
  __syncthreads();
  if (tid < SSD_Q) {
    double last = 0.0;
#pragma unroll
    for (int k = 0; k < SSD_Q / 32; k++) {
      if (k < warp) c += part_s[k];
      last += part_s[k];
    }
    w_s[tid] = exp2f((float)(last - c)) * d;
    if (v0 == 0) {
      float* sums = p.chunk_sums + (chunk * p.H + h) * 3 * SSD_Q;
      const float hi = (float)c;
      sums[tid] = d;
      sums[SSD_Q + tid] = hi;
      sums[2 * SSD_Q + tid] = (float)(c - (double)hi);
      if (tid == 0) p.chunk_decay[chunk * p.H + h] = exp2f((float)last);
    }
  }
  __syncthreads();
  if (p.vec) {
#pragma unroll
    for (int k = 0; k < XI; k++) {
      const int i = k * 256 + tid, r = i / (SSD_VB / 8), cc = (i % (SSD_VB / 8)) * 8;
      const float w = w_s[r];
      const __nv_bfloat162* x2 = (const __nv_bfloat162*)&xv[k];
      uint4 q[3];
      uint32_t* q0 = (uint32_t*)&q[0];
      uint32_t* q1 = (uint32_t*)&q[1];
      uint32_t* q2 = (uint32_t*)&q[2];
#pragma unroll
      for (int e = 0; e < 4; e++) split3_pair(w * __low2float(x2[e]), w * __high2float(x2[e]), q0[e], q1[e], q2[e]);
#pragma unroll
      for (int part = 0; part < 3; part++) *(uint4*)(Xs + (part * SSD_Q + r) * SSD_VS + cc) = q[part];
    }
  } else {
    for (int i = tid; i < SSD_Q * (SSD_VB / 2); i += 256) {
      const int r = i / (SSD_VB / 2), cc = (i % (SSD_VB / 2)) * 2;
      float u = 0.f, v = 0.f;
      if (r < n && cc < vn) {
        u = w_s[r] * to_f32(xr[(size_t)r * p.ldx + cc]);
        v = cc + 1 < vn ? w_s[r] * to_f32(xr[(size_t)r * p.ldx + cc + 1]) : 0.f;
      }
      uint32_t q0, q1, q2;
      split3_pair(u, v, q0, q1, q2);
      *(uint32_t*)(Xs + r * SSD_VS + cc) = q0;
      *(uint32_t*)(Xs + (SSD_Q + r) * SSD_VS + cc) = q1;
      *(uint32_t*)(Xs + (2 * SSD_Q + r) * SSD_VS + cc) = q2;
    }
  }
  cp_wait();
  __syncthreads();
  float* dst = p.chunk_state + (chunk * p.H + h) * (size_t)p.N * p.V;
  const int ksteps = (n + 15) / 16;
  for (int mt = warp; mt < NP / 16; mt += 8) {
    if (mt * 16 >= p.N) break;
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
      const int cc = i * 8 + (lane & 3) * 2;
      if (p.vec) {
        if (cc < vn && ra < p.N) *(float2*)(dst + (size_t)ra * p.V + v0 + cc) = make_float2(acc[i][0], acc[i][1]);
        if (cc < vn && rb < p.N) *(float2*)(dst + (size_t)rb * p.V + v0 + cc) = make_float2(acc[i][2], acc[i][3]);
      } else {
#pragma unroll
        for (int e = 0; e < 4; e++) {
          const int r = e < 2 ? ra : rb, q = cc + (e & 1);
          if (q < vn && r < p.N) dst[(size_t)r * p.V + v0 + q] = acc[i][e];
        }
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
  constexpr int AHEAD = 8;
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
template <int NP>
__global__ void __launch_bounds__(256, NP <= 128 ? 2 : 1) ssd_chunk_scan_kernel(Args p) {
  extern __shared__ __align__(16) bf16 smb[];
  __shared__ __align__(16) float sums_s[3 * SSD_Q];
  constexpr int NS = NP + 8;
  const int b = blockIdx.z, start = p.seq_start[b], len = p.seq_start[b + 1] - start;
  const int r0 = blockIdx.x * SSD_Q;
  if (r0 >= len) return;
  const int n = min(SSD_Q, len - r0), row = start + r0, tid = threadIdx.x;
  const int vblocks = (p.V + SSD_VB - 1) / SSD_VB;
  const int h = blockIdx.y / vblocks, v0 = (blockIdx.y % vblocks) * SSD_VB, g = h / (p.H / p.G), vn = min(SSD_VB, p.V - v0);
  bf16* Cs = smb;                        // [Q][NS]
  bf16* Ss = Cs + SSD_Q * NS;            // 3 x [NP][VS], later
  bf16* Bs = Ss;                         // [Q][NS]
  bf16* Xs = Bs + SSD_Q * NS;            // [Q][VS]
  const float *dt_s = sums_s, *hi = sums_s + SSD_Q, *lo = sums_s + 2 * SSD_Q;
  const bf16* xbc = (const bf16*)p.xbc + (size_t)row * p.ldx;
  const bf16* bsrc = xbc + (size_t)p.H * p.V + (size_t)g * p.N;
  const int warp = tid >> 5, lane = tid & 31, gr = lane >> 2, t = lane & 3;
  const size_t chunk = first_chunk(start, b) + blockIdx.x;
  const bool work = warp * 16 < n;
  const int ia = warp * 16 + gr, ib = ia + 8;
  stage_rows<NP>(Cs, bsrc + (size_t)p.G * p.N, p.ldx, n, p.N, p.vec);
  {
    const float* st = p.chunk_state + (chunk * p.H + h) * (size_t)p.N * p.V + v0;
    constexpr int SI = NP * (SSD_VB / 4) / 256, AT = SI < 8 ? SI : 8;      // four columns of a state row at a time, AT loads on their way
    if (p.vec) {
#pragma unroll 1
      for (int k0 = 0; k0 < SI; k0 += AT) {
        float4 q[AT];
#pragma unroll
        for (int k = 0; k < AT; k++) {
          const int i = (k0 + k) * 256 + tid, r = i / (SSD_VB / 4), c = (i % (SSD_VB / 4)) * 4;
          q[k] = r < p.N && c < vn ? *(const float4*)(st + (size_t)r * p.V + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int k = 0; k < AT; k++) {
          const int i = (k0 + k) * 256 + tid, r = i / (SSD_VB / 4), c = (i % (SSD_VB / 4)) * 4;
          uint2 s0, s1, s2;
          split3_pair(q[k].x, q[k].y, s0.x, s1.x, s2.x);
          split3_pair(q[k].z, q[k].w, s0.y, s1.y, s2.y);
          *(uint2*)(Ss + r * SSD_VS + c) = s0;
          *(uint2*)(Ss + (NP + r) * SSD_VS + c) = s1;
          *(uint2*)(Ss + (2 * NP + r) * SSD_VS + c) = s2;
        }
      }
    } else {
      for (int i = tid; i < NP * (SSD_VB / 2); i += 256) {
        const int r = i / (SSD_VB / 2), c = (i % (SSD_VB / 2)) * 2;
        const float u = r < p.N && c < vn ? st[(size_t)r * p.V + c] : 0.f, v = r < p.N && c + 1 < vn ? st[(size_t)r * p.V + c + 1] : 0.f;
        uint32_t q0, q1, q2;
        split3_pair(u, v, q0, q1, q2);
        *(uint32_t*)(Ss + r * SSD_VS + c) = q0;
        *(uint32_t*)(Ss + (NP + r) * SSD_VS + c) = q1;
        *(uint32_t*)(Ss + (2 * NP + r) * SSD_VS + c) = q2;
      }
    }
  }
  for (int i = tid; i < 3 * SSD_Q; i += 256) sums_s[i] = p.chunk_sums[(chunk * p.H + h) * 3 * SSD_Q + i];
  uint32_t zv[SSD_VB / 8][2];            // the gates of this lane's elements, on their way while the products run
  if (p.vec && work) {
    const bf16* z = (const bf16*)p.z + (size_t)row * p.ldz + (size_t)h * p.V + v0;
#pragma unroll
    for (int i = 0; i < SSD_VB / 8; i++) {
      const int c = i * 8 + 2 * t;
      zv[i][0] = c < vn && ia < n ? *(const uint32_t*)(z + (size_t)ia * p.ldz + c) : 0u;
      zv[i][1] = c < vn && ib < n ? *(const uint32_t*)(z + (size_t)ib * p.ldz + c) : 0u;
    }
  }
  cp_wait();
  __syncthreads();
  float acc[SSD_VB / 8][4];
#pragma unroll
  for (int i = 0; i < SSD_VB / 8; i++) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  const bf16* crow = Cs + (warp * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * NS + (lane >> 4) * 8;
  const float hia = hi[ia], loa = lo[ia], hib = hi[ib], lob = lo[ib];
  if (work) {
#pragma unroll 2
    for (int ks = 0; ks < NP / 16; ks++) {
      uint32_t a[4];
      ldsm4(a, crow + ks * 16);
#pragma unroll
      for (int part = 0; part < 3; part++) {
        const bf16* s = Ss + (part * NP + ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * SSD_VS + (lane >> 4) * 8;
#pragma unroll
        for (int nt = 0; nt < SSD_VB / 16; nt++) {
          uint32_t q[4];
          ldsm4t(q, s + nt * 16);
          mma_bf16(acc[2 * nt], a, q[0], q[1]);
          mma_bf16(acc[2 * nt + 1], a, q[2], q[3]);
        }
      }
    }
    const float ea = exp2f(hia + loa), eb = exp2f(hib + lob);
#pragma unroll
    for (int i = 0; i < SSD_VB / 8; i++) { acc[i][0] *= ea; acc[i][1] *= ea; acc[i][2] *= eb; acc[i][3] *= eb; }
  }
  __syncthreads();                       // the state's tile has been read
  stage_rows<NP>(Bs, bsrc, p.ldx, n, p.N, p.vec);
  stage_rows<SSD_VB>(Xs, xbc + (size_t)h * p.V + v0, p.ldx, n, vn, p.vec);
  cp_wait();
  __syncthreads();
  if (!work) return;
  for (int jt = 0; jt <= warp; jt++) {
    float gm[2][4];
#pragma unroll
    for (int i = 0; i < 2; i++) gm[i][0] = gm[i][1] = gm[i][2] = gm[i][3] = 0.f;
    const bf16* brow = Bs + (jt * 16 + (lane & 7) + (lane >> 4) * 8) * NS + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int ks = 0; ks < NP / 16; ks++) {
      uint32_t a[4], q[4];
      ldsm4(a, crow + ks * 16);
      ldsm4(q, brow + ks * 16);
      mma_bf16(gm[0], a, q[0], q[1]);
      mma_bf16(gm[1], a, q[2], q[3]);
    }
    uint32_t w[3][4];                    // the weights as A operands: halves of 8 rows j, three parts
#pragma unroll
    for (int half = 0; half < 2; half++) {
      const int j = jt * 16 + half * 8 + 2 * t;
      const float2 hj = *(const float2*)(hi + j), lj = *(const float2*)(lo + j), dj = *(const float2*)(dt_s + j);
      float wa0 = gm[half][0] * (exp2f((hia - hj.x) + (loa - lj.x)) * dj.x), wa1 = gm[half][1] * (exp2f((hia - hj.y) + (loa - lj.y)) * dj.y);
      float wb0 = gm[half][2] * (exp2f((hib - hj.x) + (lob - lj.x)) * dj.x), wb1 = gm[half][3] * (exp2f((hib - hj.y) + (lob - lj.y)) * dj.y);
      if (jt == warp) {                  // the tile on the diagonal: later rows have no say
        if (j > ia) wa0 = 0.f;
        if (j + 1 > ia) wa1 = 0.f;
        if (j > ib) wb0 = 0.f;
        if (j + 1 > ib) wb1 = 0.f;
      }
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
      bf16* o = (bf16*)p.out + (size_t)(row + r) * p.ldo + col;
      float z0, z1 = 0.f;
      if (p.vec) {
        const __nv_bfloat162 q = *(const __nv_bfloat162*)&zv[i][s];
        z0 = __low2float(q); z1 = __high2float(q);
      } else {
        const bf16* z = (const bf16*)p.z + (size_t)(row + r) * p.ldz + col;
        z0 = to_f32(z[0]);
        if (two) z1 = to_f32(z[1]);
      }
      const __nv_bfloat162 x = *(const __nv_bfloat162*)(Xs + r * SSD_VS + c);
      const float u0 = fmaf(dsk, __low2float(x), acc[i][2 * s]) * silu_fast(z0);
      const float u1 = two ? fmaf(dsk, __high2float(x), acc[i][2 * s + 1]) * silu_fast(z1) : 0.f;
      if (s) ssb += u0 * u0 + u1 * u1; else ssa += u0 * u0 + u1 * u1;
      const __nv_bfloat162 y = __floats2bfloat162_rn(u0 * w0, u1 * w1);
      if (p.vec) *(__nv_bfloat162*)o = y;
      else {
        o[0] = __low2bfloat16(y);
        if (two) o[1] = __high2bfloat16(y);
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

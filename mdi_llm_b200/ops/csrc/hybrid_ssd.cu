// State-space recurrence with one scalar decay per head and token (state-space duality), and the gated norm behind it.
//
//   dt = softplus(dt_raw + dt_bias),  a = exp(-exp(A_log) dt)
//   S <- a S + dt B x^T,   y = S^T C + D x        S [N, V] fp32 per head and slot; B, C [N] shared by a group of heads
//
// x, B, C arrive side by side in one row [H * V | G * N | G * N] (the activated convolution output); dt_raw is a column
// slice of the input projection.  Same batch conventions as hybrid_mixers.cu: meta[4*s] = {first token row, token count,
// slot, position of the first token}.  Two forms:
//
//  * ssd_scan_kernel: token by token, state in registers; one-token steps, short portions, and the 32-bit mode.
//  * ssd_chunk_state / ssd_chunk_scan / ssd_chunk_out: prompts with 16-bit activations, parallel over chunks of CL tokens.
//    With c_t the running sum of log a inside a chunk and S0 the state before it,
//      y_t = exp(c_t) S0^T C_t + sum_{s <= t} exp(c_t - c_s) dt_s (C_t . B_s) x_s + D x_t
//      S'  = exp(c_last) S0 + sum_s exp(c_last - c_s) dt_s B_s x_s^T
//    so a chunk is four small matrix products.  They run on the tensor cores: x, B, C are bf16 as they come, everything
//    fp32 that meets them (weights, states) enters as a bf16 number plus its bf16 remainder, sums are fp32.  Running
//    sums of log a are kept as a pair of floats: only differences of them are exponentiated, and those are never positive.
#include "hybrid_mma.cuh"

namespace hyb {

struct SsdArgs {
  const void *xbc, *dt;              // [tokens][xbc_stride], [tokens][dt_stride]
  const float *dt_bias, *a_log, *d;  // [H]
  float* state;                      // [slots][H][N][V]
  float* y;                          // [tokens][H * V]
  const int *meta, *ctab, *stab;     // chunk c: {first token row, tokens, sequence, 0}; sequence: {first chunk, chunks}
  float* u;                          // [chunks][H][N][V]: what a chunk adds to the state
  float* decay;                      // [chunks][H]: exp(c_last)
  void* before;                      // [chunks][H][2][N][V] bf16: the state before a chunk, rounded, and the remainder
  long long xbc_stride, dt_stride;
  int H, G, N, V, nseq, nchunks;
};

// Block = (sequence, head, 32 value columns): lane = column, warp w owns the state rows w, w + 8, ..
#define SS_MAXI 32
template <typename T, int MAXI>
__global__ void __launch_bounds__(256) ssd_scan_kernel(SsdArgs a) {
  __shared__ float bs[256], cs[256], part[8][33];
  const int* m = a.meta + 4 * blockIdx.x;
  const int r0 = m[0], n = m[1], h = blockIdx.y, lane = threadIdx.x & 31, w = threadIdx.x >> 5;
  const int vc = blockIdx.z * 32 + lane, N = a.N, V = a.V;
  const bool live = vc < V;
  const int g = h / (a.H / a.G);
  float* sp = a.state + ((size_t)m[2] * a.H + h) * N * V;
  const T* row = (const T*)a.xbc + (size_t)r0 * a.xbc_stride;
  const T* dr = (const T*)a.dt + (size_t)r0 * a.dt_stride + h;
  const float bias = a.dt_bias[h], rate = expf(a.a_log[h]), skip = a.d[h];
  float S[MAXI];
#pragma unroll
  for (int i = 0; i < MAXI; ++i) {
    int d = w + 8 * i;
    S[i] = d < N && live ? sp[(size_t)d * V + vc] : 0.f;
  }
  for (int t = 0; t < n; ++t, row += a.xbc_stride, dr += a.dt_stride) {
    for (int d = threadIdx.x; d < N; d += 256) {
      bs[d] = to_f(row[(size_t)a.H * V + g * N + d]);
      cs[d] = to_f(row[(size_t)a.H * V + (a.G + g) * N + d]);
    }
    const float dt = softplusf_(to_f(dr[0]) + bias), al = expf(-rate * dt);
    const float x = live ? to_f(row[(size_t)h * V + vc]) : 0.f, dx = dt * x;
    __syncthreads();
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < MAXI; ++i) {
      int d = w + 8 * i;
      if (d < N) {
        S[i] = al * S[i] + bs[d] * dx;
        o += S[i] * cs[d];
      }
    }
    part[w][lane] = o;
    __syncthreads();
    if (w == 0 && live) {
      float y = skip * x;
#pragma unroll
      for (int i = 0; i < 8; ++i) y += part[i][lane];
      a.y[(size_t)(r0 + t) * a.H * V + (size_t)h * V + vc] = y;
    }
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < MAXI; ++i) {
      int d = w + 8 * i;
      if (d < N) sp[(size_t)d * V + vc] = S[i];
    }
  }
}

// c = a + b with the rounding error of the sum kept in the second component
__device__ __forceinline__ float2 pair_add(float2 a, float2 b) {
  float s = a.x + b.x, t = s - a.x;
  float e = (a.x - (s - t)) + (b.x - t) + (a.y + b.y);
  float r = s + e;
  return make_float2(r, e - (r - s));
}
__device__ __forceinline__ float pair_diff(float2 a, float2 b) { return (a.x - b.x) + (a.y - b.y); }

// dts[s] = dt of the chunk's token s, cum[s] = log a_0 + .. + log a_s; tokens from len on: dt 0, log a 0.  One warp.
template <int CL>
__device__ __forceinline__ void chunk_decays(const SsdArgs& a, int row0, int len, int h, int lane, float* dts, float2* cum) {
  const float bias = a.dt_bias[h], rate = expf(a.a_log[h]);
  float2 carry = make_float2(0.f, 0.f);
  for (int s0 = 0; s0 < CL; s0 += 32) {
    const int s = s0 + lane;
    float dt = 0.f;
    if (s < len) dt = softplusf_(to_f(((const bf16*)a.dt)[(size_t)(row0 + s) * a.dt_stride + h]) + bias);
    float2 c = make_float2(-rate * dt, 0.f);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      float2 p = make_float2(__shfl_up_sync(0xffffffffu, c.x, o), __shfl_up_sync(0xffffffffu, c.y, o));
      if (lane >= o) c = pair_add(c, p);
    }
    c = pair_add(carry, c);
    dts[s] = dt;
    cum[s] = c;
    carry = make_float2(__shfl_sync(0xffffffffu, c.x, 31), __shfl_sync(0xffffffffu, c.y, 31));
  }
}

// rows [0, rows) x columns [0, cols) of a bf16 matrix into shared memory with row length ld; columns up to `colsp` and
// rows from `live` on become zero.  vec: 16-byte asynchronous copies (cols a multiple of 8, sources 16-byte aligned).
template <int TH>
__device__ __forceinline__ void stage(bf16* dst, int ld, const bf16* src, long long stride, int rows, int live, int cols, int colsp, int vec) {
  if (vec) {
    const int per = colsp >> 3;
    for (int i = threadIdx.x; i < rows * per; i += TH) {
      int r = i / per, c = (i - r * per) * 8;
      bool ok = r < live && c < cols;
      cp16(dst + r * ld + c, ok ? src + (size_t)r * stride + c : src, ok);
    }
    return;
  }
  for (int i = threadIdx.x; i < rows * colsp; i += TH) {
    int r = i / colsp, c = i - r * colsp;
    dst[r * ld + c] = r < live && c < cols ? src[(size_t)r * stride + c] : __float2bfloat16_rn(0.f);
  }
}

// U = sum_s B_s (w_s x_s)^T, w_s = exp(c_last - c_s) dt_s.  Block = (chunk, head), 4 warps; warp w owns the state rows of
// the 16-row tiles w, w + 4, ..; value columns in tiles of 64, the weighted x as number plus remainder.
template <int CL>
__global__ void __launch_bounds__(128) ssd_chunk_state_kernel(SsdArgs a, int vec) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float dts[CL];
  __shared__ float2 cum[CL];
  const int N = a.N, V = a.V, Np = (N + 15) & ~15, ldn = Np + 8, ldv = 64 + 8;
  bf16* bs = reinterpret_cast<bf16*>(raw);  // [CL][ldn]
  bf16* xh = bs + CL * ldn;                 // [CL][ldv]
  bf16* xl = xh + CL * ldv;                 // [CL][ldv]
  const int* c = a.ctab + 4 * blockIdx.x;
  const int row0 = c[0], len = c[1], h = blockIdx.y, g = h / (a.H / a.G);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, t2 = (lane & 3) * 2;
  const bf16* base = (const bf16*)a.xbc + (size_t)row0 * a.xbc_stride;
  stage<128>(bs, ldn, base + (size_t)a.H * V + (size_t)g * N, a.xbc_stride, CL, len, N, Np, vec);
  cp_commit();
  if (warp == 0) chunk_decays<CL>(a, row0, len, h, lane, dts, cum);
  __syncthreads();
  if (tid == 0) a.decay[(size_t)blockIdx.x * a.H + h] = expf(cum[CL - 1].x + cum[CL - 1].y);
  for (int s = tid; s < CL; s += 128) dts[s] *= expf(pair_diff(cum[CL - 1], cum[s]));
  float* up = a.u + ((size_t)blockIdx.x * a.H + h) * N * V;
  for (int v0 = 0; v0 < V; v0 += 64) {
    const int cols = min(64, V - v0), colsp = (cols + 15) & ~15;
    __syncthreads();  // weights are final; the tile before is done with xh, xl
    if (vec) {
      const int per = colsp >> 3;
      for (int i = tid; i < CL * per; i += 128) {
        int s = i / per, cc = (i - s * per) * 8;
        float f[8], lo[8];
        if (s < len && cc < cols) {
          load8(base + (size_t)s * a.xbc_stride + (size_t)h * V + v0 + cc, f);
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = 0.f;
        }
        const float w = dts[s];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          f[e] *= w;
          lo[e] = f[e] - __bfloat162float(__float2bfloat16_rn(f[e]));
        }
        store8(xh + s * ldv + cc, f);
        store8(xl + s * ldv + cc, lo);
      }
    } else {
      for (int i = tid; i < CL * colsp; i += 128) {
        int s = i / colsp, cc = i - s * colsp;
        float f = s < len && cc < cols ? dts[s] * to_f(base[(size_t)s * a.xbc_stride + (size_t)h * V + v0 + cc]) : 0.f;
        bf16 hi = __float2bfloat16_rn(f);
        xh[s * ldv + cc] = hi;
        xl[s * ldv + cc] = __float2bfloat16_rn(f - __bfloat162float(hi));
      }
    }
    cp_wait<0>();
    __syncthreads();
    const int nv = colsp >> 4;
    for (int d0 = warp * 16; d0 < Np; d0 += 64) {
      float acc[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
      for (int k = 0; k < CL; k += 16) {
        uint32_t A[4];  // A[d][s] = B[s][d]: transposed 8x8 blocks (d 0-7 | 8-15) x (s 0-7 | 8-15)
        ldm4t(A, bs + (k + (lane & 7) + (lane >> 4) * 8) * ldn + d0 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (i < nv) {
            uint32_t b[4];
            ldm4t(b, xh + (k + (lane & 15)) * ldv + i * 16 + (lane >> 4) * 8);
            mma(acc[2 * i], A, b);
            mma(acc[2 * i + 1], A, b + 2);
            ldm4t(b, xl + (k + (lane & 15)) * ldv + i * 16 + (lane >> 4) * 8);
            mma(acc[2 * i], A, b);
            mma(acc[2 * i + 1], A, b + 2);
          }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          int d = d0 + gr + 8 * r, cc = i * 8 + t2;
          if (d >= N || cc >= cols) continue;
          float* p = up + (size_t)d * V + v0 + cc;
          if (vec) {
            *reinterpret_cast<float2*>(p) = make_float2(acc[i][2 * r], acc[i][2 * r + 1]);
          } else {
            p[0] = acc[i][2 * r];
            if (cc + 1 < cols) p[1] = acc[i][2 * r + 1];
          }
        }
    }
  }
}

// Walks a sequence's chunks: before[c] = S (number and remainder), S = decay_c S + U_c; the slot keeps the final S.
// VEC neighbouring elements of the [N, V] state per thread, the U of eight chunks in flight.
template <int VEC>
__global__ void __launch_bounds__(256) ssd_chunk_scan_kernel(SsdArgs a) {
  const int seq = blockIdx.x, h = blockIdx.y, NV = a.N * a.V;
  const int slot = a.meta[4 * seq + 2], c0 = a.stab[2 * seq], nc = a.stab[2 * seq + 1];
  const int e = (blockIdx.z * 256 + threadIdx.x) * VEC;
  if (e >= NV) return;
  float* sp = a.state + ((size_t)slot * a.H + h) * NV + e;
  const float* u = a.u + ((size_t)c0 * a.H + h) * NV + e;
  bf16* bf = (bf16*)a.before + ((size_t)c0 * a.H + h) * 2 * NV + e;
  const float* dc = a.decay + (size_t)c0 * a.H + h;
  const size_t cs = (size_t)a.H * NV;
  float S[VEC];
#pragma unroll
  for (int k = 0; k < VEC; ++k) S[k] = sp[k];
  for (int c = 0; c < nc; c += 8) {
    float U[8][VEC], D[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const bool ok = c + i < nc;
      D[i] = ok ? dc[(size_t)(c + i) * a.H] : 0.f;
      if (VEC == 4) {
        float4 f = ok ? *reinterpret_cast<const float4*>(u + (size_t)(c + i) * cs) : make_float4(0.f, 0.f, 0.f, 0.f);
        U[i][0] = f.x; U[i][1] = f.y; U[i][2] = f.z; U[i][3] = f.w;
      } else {
        U[i][0] = ok ? u[(size_t)(c + i) * cs] : 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (c + i < nc) {
        bf16* b = bf + (size_t)(c + i) * 2 * cs;
        if (VEC == 4) {
          uint32_t h0, l0, h1, l1;
          split2(S[0], S[1], h0, l0);
          split2(S[2], S[3], h1, l1);
          *reinterpret_cast<uint2*>(b) = make_uint2(h0, h1);
          *reinterpret_cast<uint2*>(b + NV) = make_uint2(l0, l1);
        } else {
          bf16 hi = __float2bfloat16_rn(S[0]);
          b[0] = hi;
          b[NV] = __float2bfloat16_rn(S[0] - __bfloat162float(hi));
        }
#pragma unroll
        for (int k = 0; k < VEC; ++k) S[k] = D[i] * S[k] + U[i][k];
      }
    }
  }
#pragma unroll
  for (int k = 0; k < VEC; ++k) sp[k] = S[k];
}

// y of a chunk.  Block = (chunk, head), CL / 16 warps of 16 token rows; value columns in tiles of 64.  Per row: first the
// read-out of the state before the chunk, scaled by exp(c_t), then tile by tile of 16 earlier tokens the products C.B,
// weighed in registers and multiplied into x.
template <int CL>
__global__ void __launch_bounds__(2 * CL) ssd_chunk_out_kernel(SsdArgs a, int vec) {
  constexpr int TH = 2 * CL;
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float dts[CL];
  __shared__ float2 cum[CL];
  const int N = a.N, V = a.V, Np = (N + 15) & ~15, ldn = Np + 8, ldv = 64 + 8;
  bf16* cm = reinterpret_cast<bf16*>(raw);  // [CL][ldn]
  bf16* bs = cm + CL * ldn;                 // [CL][ldn]
  bf16* xs = bs + CL * ldn;                 // [CL][ldv]
  bf16* sh = xs + CL * ldv;                 // [Np][ldv]
  bf16* sl = sh + Np * ldv;                 // [Np][ldv]
  const int* c = a.ctab + 4 * blockIdx.x;
  const int row0 = c[0], len = c[1], h = blockIdx.y, g = h / (a.H / a.G);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, t2 = (lane & 3) * 2;
  const bf16* base = (const bf16*)a.xbc + (size_t)row0 * a.xbc_stride;
  const bf16* before = (const bf16*)a.before + ((size_t)blockIdx.x * a.H + h) * 2 * N * V;
  stage<TH>(cm, ldn, base + (size_t)a.H * V + (size_t)(a.G + g) * N, a.xbc_stride, CL, len, N, Np, vec);
  stage<TH>(bs, ldn, base + (size_t)a.H * V + (size_t)g * N, a.xbc_stride, CL, len, N, Np, vec);
  const int r0 = warp * 16;  // this lane's rows: r0 + gr and r0 + gr + 8
  const float skip = a.d[h];
  for (int v0 = 0; v0 < V; v0 += 64) {
    const int cols = min(64, V - v0), colsp = (cols + 15) & ~15, nv = colsp >> 4;
    __syncthreads();  // the tile before is done with xs, sh, sl
    stage<TH>(xs, ldv, base + (size_t)h * V + v0, a.xbc_stride, CL, len, cols, colsp, vec);
    stage<TH>(sh, ldv, before + v0, V, Np, N, cols, colsp, vec);
    stage<TH>(sl, ldv, before + (size_t)N * V + v0, V, Np, N, cols, colsp, vec);
    cp_commit();
    if (v0 == 0 && warp == 0) chunk_decays<CL>(a, row0, len, h, lane, dts, cum);
    cp_wait<0>();
    __syncthreads();
    if (r0 < len) {
      float acc[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
      const bf16* ap = cm + (r0 + (lane & 15)) * ldn + (lane >> 4) * 8;
      for (int k = 0; k < Np; k += 16) {
        uint32_t A[4], b[4];
        ldm4(A, ap + k);
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (i < nv) {
            ldm4t(b, sh + (k + (lane & 15)) * ldv + i * 16 + (lane >> 4) * 8);
            mma(acc[2 * i], A, b);
            mma(acc[2 * i + 1], A, b + 2);
            ldm4t(b, sl + (k + (lane & 15)) * ldv + i * 16 + (lane >> 4) * 8);
            mma(acc[2 * i], A, b);
            mma(acc[2 * i + 1], A, b + 2);
          }
      }
      const float2 ct[2] = {cum[r0 + gr], cum[r0 + gr + 8]};
      const float e0 = expf(ct[0].x + ct[0].y), e1 = expf(ct[1].x + ct[1].y);
#pragma unroll
      for (int i = 0; i < 8; ++i) { acc[i][0] *= e0; acc[i][1] *= e0; acc[i][2] *= e1; acc[i][3] *= e1; }
      for (int s0 = 0; s0 <= r0; s0 += 16) {
        float s[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
        const bf16* bp = bs + (s0 + (lane & 7) + (lane >> 4) * 8) * ldn + ((lane >> 3) & 1) * 8;
#pragma unroll 4
        for (int k = 0; k < Np; k += 16) {
          uint32_t A[4], b[4];
          ldm4(A, ap + k);
          ldm4(b, bp + k);
          mma(s[0], A, b);
          mma(s[1], A, b + 2);
        }
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int src = s0 + u * 8 + t2 + (e & 1), row = r0 + gr + (e >> 1) * 8;
            s[u][e] = src <= row ? s[u][e] * (dts[src] * expf(pair_diff(ct[e >> 1], cum[src]))) : 0.f;
          }
          split2(s[u][0], s[u][1], hi[2 * u], lo[2 * u]);
          split2(s[u][2], s[u][3], hi[2 * u + 1], lo[2 * u + 1]);
        }
        const bf16* xp = xs + (s0 + (lane & 15)) * ldv + (lane >> 4) * 8;
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (i < nv) {
            uint32_t b[4];
            ldm4t(b, xp + i * 16);
            mma(acc[2 * i], hi, b);
            mma(acc[2 * i + 1], hi, b + 2);
            mma(acc[2 * i], lo, b);
            mma(acc[2 * i + 1], lo, b + 2);
          }
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int row = r0 + gr + 8 * r;
        if (row >= len) continue;
        float* yp = a.y + (size_t)(row0 + row) * a.H * V + (size_t)h * V + v0;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int cc = i * 8 + t2;
          if (cc >= cols) continue;
          const float y0 = acc[i][2 * r] + skip * to_f(xs[row * ldv + cc]), y1 = acc[i][2 * r + 1] + skip * to_f(xs[row * ldv + cc + 1]);
          if (vec) {
            *reinterpret_cast<float2*>(yp + cc) = make_float2(y0, y1);
          } else {
            yp[cc] = y0;
            if (cc + 1 < cols) yp[cc + 1] = y1;
          }
        }
      }
    }
  }
}

// out = w * (y silu(z)) / rms over each of `parts` equal parts of the row.  Block = (row, part); the gated part waits in
// shared memory for its root mean square.
template <typename T, int VEC>
__global__ void silu_gate_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, long long z_stride,
                                      const T* __restrict__ w, T* __restrict__ out, int n, int per, float eps) {
  extern __shared__ __align__(16) float buf[];  // [per]
  __shared__ float red[33];
  const size_t r = blockIdx.x;
  const int c0 = blockIdx.y * per;
  const float* yr = y + r * n + c0;
  const T* zr = z + r * z_stride + c0;
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < per; i += blockDim.x * VEC) {
    float f[VEC], g[VEC];
    if (VEC == 8) { load8(yr + i, f); load8(zr + i, g); }
    else { f[0] = yr[i]; g[0] = to_f(zr[i]); }
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      f[e] *= siluf_(g[e]);
      ss += f[e] * f[e];
    }
    if (VEC == 8) store8(buf + i, f);
    else buf[i] = f[0];
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / per + eps);
  for (int i = threadIdx.x * VEC; i < per; i += blockDim.x * VEC) {  // a thread reads what it has written
    float f[VEC], g[VEC];
    if (VEC == 8) { load8(buf + i, f); load8(w + c0 + i, g); }
    else { f[0] = buf[i]; g[0] = to_f(w[c0 + i]); }
#pragma unroll
    for (int e = 0; e < VEC; ++e) f[e] *= inv * g[e];
    if (VEC == 8) store8(out + r * n + c0 + i, f);
    else out[r * n + c0 + i] = from_f<T>(f[0]);
  }
}

}  // namespace hyb

using namespace hyb;

extern "C" {

// The token scan.  -3: more than 256 state rows.
int hyb_ssd_scan(const SsdArgs* args, int dt, cudaStream_t st) {
  const SsdArgs& a = *args;
  if (a.nseq == 0) return 0;
  if (a.G < 1 || a.H % a.G || a.N < 1 || a.V < 1) return -2;
  if (a.N > 8 * SS_MAXI) return -3;
  dim3 grid(a.nseq, a.H, (a.V + 31) / 32);
#define SC(T) do { if (a.N <= 64) ssd_scan_kernel<T, 8><<<grid, 256, 0, st>>>(a); else if (a.N <= 128) ssd_scan_kernel<T, 16><<<grid, 256, 0, st>>>(a); \
                   else ssd_scan_kernel<T, SS_MAXI><<<grid, 256, 0, st>>>(a); } while (0)
  if (dt == 0) SC(bf16); else SC(float);
#undef SC
  return (int)cudaGetLastError();
}

// Shared memory of the output kernel for chunks of `cl` tokens (the largest of the three); 0: no such kernel.
static size_t ssd_out_smem(int cl, int N) {
  size_t Np = (size_t)((N + 15) & ~15);
  return (2 * cl * (Np + 8) + (size_t)cl * 72 + 2 * Np * 72) * sizeof(bf16);
}

// The chunked form (bf16): -3 when the shared memory of a block does not hold the shape.
int hyb_ssd_chunked(const SsdArgs* args, int cl, cudaStream_t st) {
  const SsdArgs& a = *args;
  if (a.nseq == 0) return 0;
  if (a.G < 1 || a.H % a.G || a.N < 1 || a.V < 1 || (cl != 64 && cl != 128)) return -2;
  const size_t so = ssd_out_smem(cl, a.N), ss = ((size_t)cl * (((a.N + 15) & ~15) + 8) + 2 * (size_t)cl * 72) * sizeof(bf16);
  if (so > 200 * 1024 || ss > 200 * 1024 || a.H > 65535) return -3;
  const uintptr_t bits = (uintptr_t)a.xbc | (uintptr_t)a.u | (uintptr_t)a.before | (uintptr_t)a.y | (uintptr_t)a.state;
  const int vec = (bits & 15) == 0 && ((a.N | a.V) & 7) == 0 && (a.xbc_stride & 7) == 0;
  dim3 grid(a.nchunks, a.H);
#define CK(CL)                                                                                                        \
  do {                                                                                                                \
    cudaFuncSetAttribute(ssd_chunk_state_kernel<CL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ss);           \
    cudaFuncSetAttribute(ssd_chunk_out_kernel<CL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)so);             \
    ssd_chunk_state_kernel<CL><<<grid, 128, ss, st>>>(a, vec);                                                        \
    if (vec) ssd_chunk_scan_kernel<4><<<dim3(a.nseq, a.H, (a.N * a.V + 1023) / 1024), 256, 0, st>>>(a);               \
    else ssd_chunk_scan_kernel<1><<<dim3(a.nseq, a.H, (a.N * a.V + 255) / 256), 256, 0, st>>>(a);                     \
    ssd_chunk_out_kernel<CL><<<grid, 2 * CL, so, st>>>(a, vec);                                                       \
  } while (0)
  if (cl == 64) CK(64); else CK(128);
#undef CK
  return (int)cudaGetLastError();
}

int hyb_silu_gate_norm(const float* y, const void* z, long long z_stride, const void* w, void* out, int rows, int n, int parts,
                       float eps, int dt, cudaStream_t st) {
  if (rows == 0) return 0;
  if (parts < 1 || n % parts || parts > 65535) return -2;
  const int per = n / parts;
  const size_t smem = (size_t)per * sizeof(float);
  if (smem > 200 * 1024) return -3;
  const uintptr_t bits = (uintptr_t)y | (uintptr_t)z | (uintptr_t)w | (uintptr_t)out;
  const bool vec = (bits & 15) == 0 && ((n | per) & 7) == 0 && (z_stride & 7) == 0;
  const int work = vec ? per / 8 : per, th = work >= 256 ? 256 : (work + 31) / 32 * 32;
#define GN(T, V)                                                                                                            \
  do {                                                                                                                      \
    if (smem > 40 * 1024)                                                                                                   \
      cudaFuncSetAttribute(silu_gate_norm_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);            \
    silu_gate_norm_kernel<T, V><<<dim3(rows, parts), th, smem, st>>>(y, (const T*)z, z_stride, (const T*)w, (T*)out, n, per, eps); \
  } while (0)
  if (dt == 0) { if (vec) GN(bf16, 8); else GN(bf16, 1); }
  else { if (vec) GN(float, 8); else GN(float, 1); }
#undef GN
  return (int)cudaGetLastError();
}

}  // extern "C"

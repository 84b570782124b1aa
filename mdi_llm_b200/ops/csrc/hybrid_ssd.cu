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
//  * ssd_decay_kernel, ssd_walk_kernel, ssd_out_kernel: prompts with 16-bit activations, in chunks.  With c_t the running sum of log a
//    inside a chunk and S0 the state before it,
//      S'  = exp(c_last) S0 + sum_s exp(c_last - c_s) dt_s B_s x_s^T
//      y_t = exp(c_t) S0^T C_t + sum_{s <= t} exp(c_t - c_s) dt_s (C_t . B_s) x_s + D x_t
//    Only the first line chains the chunks: the walk follows it through a sequence with the state in registers and leaves
//    the state before every chunk; the second line then runs for all chunks at once.  Both are small matrix products on
//    the tensor cores: x, B, C are bf16 as they come, everything fp32 that meets them (weights, states) enters as a bf16
//    number plus its bf16 remainder, sums are fp32.  Running sums of log a are kept as a pair of floats: only differences
//    of them are exponentiated, and those are never positive.
#include "hybrid_mma.cuh"

namespace hyb {

struct SsdArgs {
  const void *xbc, *dt;              // [tokens][xbc_stride], [tokens][dt_stride]
  const float *dt_bias, *a_log, *d;  // [H]
  float* state;                      // [slots][H][N][V]
  float* y;                          // [tokens][H * V]
  const int *meta, *ctab, *stab;     // chunk of SSD_CL tokens: {first token row, tokens, sequence, 0}; sequence: {first chunk, chunks}
  void* before;                      // [chunks][H][2][N][V] bf16: the state before a chunk, rounded, and the remainder
  float4* dec;                       // [H][tokens]: {running sum of log a in its 64 tokens (two floats), dt, exp(c_last - c) dt}
  long long xbc_stride, dt_stride;
  int H, G, N, V, nseq, nchunks, tokens;
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

// Step sizes and decays of 64 tokens at a time (the steps of the walk), one warp per 64 tokens and head: dt, the running sum
// c of log a, and what weighs a token in the state after the 64: exp(c_last - c) dt.
#define SW_L 64
#define SSD_CL 128  // tokens per chunk of the outputs: the state before every second step of the walk is written out
__global__ void __launch_bounds__(256) ssd_decay_kernel(SsdArgs a) {
  const int* ch = a.ctab + 4 * blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, piece = warp & 1, h = blockIdx.y * 4 + (warp >> 1);
  const int row0 = ch[0] + piece * SW_L, len = min(SW_L, ch[1] - piece * SW_L);
  if (h >= a.H || len <= 0) return;
  const float bias = a.dt_bias[h], rate = expf(a.a_log[h]);
  float dt[2];
  float2 c[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int s = lane + 32 * i;
    dt[i] = s < len ? softplusf_(to_f(((const bf16*)a.dt)[(size_t)(row0 + s) * a.dt_stride + h]) + bias) : 0.f;
    c[i] = make_float2(-rate * dt[i], 0.f);
  }
#pragma unroll
  for (int k = 1; k < 32; k <<= 1)
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      float2 p = make_float2(__shfl_up_sync(0xffffffffu, c[i].x, k), __shfl_up_sync(0xffffffffu, c[i].y, k));
      if (lane >= k) c[i] = pair_add(c[i], p);
    }
  c[1] = pair_add(make_float2(__shfl_sync(0xffffffffu, c[0].x, 31), __shfl_sync(0xffffffffu, c[0].y, 31)), c[1]);
  const float2 last = make_float2(__shfl_sync(0xffffffffu, c[1].x, 31), __shfl_sync(0xffffffffu, c[1].y, 31));
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int s = lane + 32 * i;
    if (s < len) a.dec[(size_t)h * a.tokens + row0 + s] = make_float4(c[i].x, c[i].y, dt[i], dt[i] * expf(pair_diff(last, c[i])));
  }
}

// rows [0, rows) x columns [0, cols) of a bf16 matrix into shared memory with row length ld; columns up to `colsp` and
// rows from `live` on become zero.  vec: 16-byte asynchronous copies by `rc` (cols a multiple of 8, sources 16-byte aligned).
template <int TH>
__device__ __forceinline__ void stage(const RowCopy& rc, bf16* dst, int ld, const bf16* src, long long stride, int rows, int live, int cols,
                                      int colsp, int vec) {
  if (vec) {
    rc.run(dst, ld, src, stride, rows, live, cols);
    return;
  }
  for (int i = threadIdx.x; i < rows * colsp; i += TH) {
    int r = i / colsp, c = i - r * colsp;
    dst[r * ld + c] = r < live && c < cols ? src[(size_t)r * stride + c] : __float2bfloat16_rn(0.f);
  }
}

// Block = (sequence, head, 32 value columns), 8 warps: warp w owns the state rows of the 16-row tiles w, w + 8, .. as
// accumulators in registers.  A step takes in 64 tokens.  Its rows arrive by asynchronous copies ahead of time; one step
// ahead, x is multiplied by the tokens' weights and split into a bf16 number and its remainder, the right operands.
#define SW_TH 256
#define SW_VT 32
#define SW_STAGES 4
template <int MT>
__global__ void __launch_bounds__(SW_TH) ssd_walk_kernel(SsdArgs a, int vec) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ __align__(16) float4 dec[SW_STAGES][SW_L];
  const int N = a.N, V = a.V, Np = (N + 15) & ~15, ldn = Np + 8;
  constexpr int ldv = SW_VT + 8;
  bf16* bs = reinterpret_cast<bf16*>(raw);       // [SW_STAGES][SW_L][ldn]
  bf16* xs = bs + SW_STAGES * SW_L * ldn;        // [SW_STAGES][SW_L][ldv]
  bf16* wx = xs + SW_STAGES * SW_L * ldv;        // [2][number, remainder][SW_L][ldv]
  const int* m = a.meta + 4 * blockIdx.x;
  const int first = m[0], n = m[1], h = blockIdx.y, g = h / (a.H / a.G), v0 = blockIdx.z * SW_VT;
  const int cols = min(SW_VT, V - v0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, t2 = (lane & 3) * 2;
  float* sp = a.state + ((size_t)m[2] * a.H + h) * N * V + v0;
  bf16* out = (bf16*)a.before + ((size_t)a.stab[2 * blockIdx.x] * a.H + h) * 2 * N * V + v0;
  const RowCopy rb(Np >> 3, tid, SW_TH), rx(SW_VT >> 3, tid, SW_TH);
  const bf16* bsrc = (const bf16*)a.xbc + (size_t)first * a.xbc_stride + (size_t)a.H * V + (size_t)g * N;
  const bf16* xsrc = (const bf16*)a.xbc + (size_t)first * a.xbc_stride + (size_t)h * V + v0;
  const float4* dsrc = a.dec + (size_t)h * a.tokens + first;
  auto fetch = [&](int c) {
    if (c < n) {
      const int len = min(SW_L, n - c), buf = (c / SW_L) % SW_STAGES;
      stage<SW_TH>(rb, bs + buf * SW_L * ldn, ldn, bsrc + (size_t)c * a.xbc_stride, a.xbc_stride, SW_L, len, N, Np, vec);
      stage<SW_TH>(rx, xs + buf * SW_L * ldv, ldv, xsrc + (size_t)c * a.xbc_stride, a.xbc_stride, SW_L, len, cols, SW_VT, vec);
      if (tid < SW_L) cp16(reinterpret_cast<bf16*>(&dec[buf][tid]), reinterpret_cast<const bf16*>(dsrc + c + (tid < len ? tid : 0)), tid < len);
    }
    cp_commit();  // possibly an empty group: the waits count groups
  };
  auto weigh = [&](int c) {  // 8 channels of one token per thread
    if (c >= n) return;
    const int buf = (c / SW_L) % SW_STAGES, s = tid >> 2, cc = (tid & 3) * 8;
    bf16* o = wx + ((c / SW_L) & 1) * 2 * SW_L * ldv + s * ldv + cc;
    const float w = dec[buf][s].w;
    float f[8];
    load8(xs + (buf * SW_L + s) * ldv + cc, f);
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) split2(f[2 * e] * w, f[2 * e + 1] * w, hi[e], lo[e]);
    *reinterpret_cast<uint4*>(o) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(o + SW_L * ldv) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  };
  float S[MT][SW_VT / 8][4];
  fetch(0);
  fetch(SW_L);
  fetch(2 * SW_L);
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < SW_VT / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (warp + 8 * i) * 16 + gr + 8 * (e >> 1), c = j * 8 + t2 + (e & 1);
        S[i][j][e] = d < N && c < cols ? sp[(size_t)d * V + c] : 0.f;
      }
  cp_wait<2>();
  __syncthreads();
  weigh(0);
  for (int c0 = 0; c0 < n; c0 += SW_L) {
    const int len = min(SW_L, n - c0), buf = (c0 / SW_L) % SW_STAGES;
    cp_wait<1>();     // this thread's copies of the next step
    __syncthreads();  // everybody's; and everybody is done with the step before
    fetch(c0 + 3 * SW_L);
    const bf16* bb = bs + buf * SW_L * ldn;
    const bf16* wh = wx + ((c0 / SW_L) & 1) * 2 * SW_L * ldv;
    if (c0 % SSD_CL == 0) {  // the state before this chunk of the outputs
      bf16* hi = out + (size_t)(c0 / SSD_CL) * a.H * 2 * N * V;
#pragma unroll
      for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int d = (warp + 8 * i) * 16 + gr + 8 * r;
          if (d >= N) continue;
          bf16* p = hi + (size_t)d * V + t2;
#pragma unroll
          for (int j = 0; j < SW_VT / 8; ++j) {
            const int c = j * 8 + t2;
            if (c >= cols) continue;
            uint32_t x, y;
            split2(S[i][j][2 * r], S[i][j][2 * r + 1], x, y);
            if (vec) {
              *reinterpret_cast<uint32_t*>(p + j * 8) = x;
              *reinterpret_cast<uint32_t*>(p + (size_t)N * V + j * 8) = y;
            } else {
              const __nv_bfloat162 px = *reinterpret_cast<__nv_bfloat162*>(&x), py = *reinterpret_cast<__nv_bfloat162*>(&y);
              p[j * 8] = px.x;
              p[(size_t)N * V + j * 8] = py.x;
              if (c + 1 < cols) { p[j * 8 + 1] = px.y; p[(size_t)N * V + j * 8 + 1] = py.y; }
            }
          }
        }
    }
    const float4 end = dec[buf][len - 1];
    const float all = expf(end.x + end.y);
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < SW_VT / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][j][e] *= all;
#pragma unroll
    for (int k = 0; k < SW_L; k += 16) {  // rows from len on are zero
      uint32_t b[SW_VT / 16][4], d[SW_VT / 16][4];
#pragma unroll
      for (int j = 0; j < SW_VT / 16; ++j) {
        ldm4t(b[j], wh + (k + (lane & 15)) * ldv + (lane >> 4) * 8 + j * 16);
        ldm4t(d[j], wh + (SW_L + k + (lane & 15)) * ldv + (lane >> 4) * 8 + j * 16);
      }
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        const int d0 = (warp + 8 * i) * 16;
        if (d0 >= Np) continue;
        uint32_t A[4];  // A[d][s] = B[s][d]: transposed 8x8 blocks (d 0-7 | 8-15) x (s 0-7 | 8-15)
        ldm4t(A, bb + (k + (lane & 7) + (lane >> 4) * 8) * ldn + d0 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int j = 0; j < SW_VT / 16; ++j) {
          mma(S[i][2 * j], A, b[j]);
          mma(S[i][2 * j + 1], A, b[j] + 2);
        }
#pragma unroll
        for (int j = 0; j < SW_VT / 16; ++j) {
          mma(S[i][2 * j], A, d[j]);
          mma(S[i][2 * j + 1], A, d[j] + 2);
        }
      }
    }
    weigh(c0 + SW_L);
  }
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < SW_VT / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (warp + 8 * i) * 16 + gr + 8 * (e >> 1), c = j * 8 + t2 + (e & 1);
        if (d < N && c < cols) sp[(size_t)d * V + c] = S[i][j][e];
      }
}

// y of a chunk.  Block = (chunk, head), 8 warps of 16 token rows; value columns in tiles of 64.  C stays in registers as
// left operand (NK: 16-wide steps of the state size).  With r the last token before a warp's 16 rows,
//   y_t = exp(c_t - c_r) [exp(c_r) S0^T C_t + sum_{s <= r} f(r, s) (C_t . B_s) x_s] + (the same 16 tokens, weighed one by one)
// where f(r, s) = exp(c_r - c_s) dt_s is shared by the warp's rows: a table of them is made once per block.
template <int NK>
__global__ void __launch_bounds__(2 * SSD_CL, NK <= 8 ? 2 : 1) ssd_out_kernel(SsdArgs a, int vec) {
  constexpr int TH = 2 * SSD_CL, ldv = 64 + 8;
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float2 cum[SSD_CL];
  __shared__ float dts[SSD_CL];
  __shared__ __align__(8) float tab[SSD_CL / 16][SSD_CL];  // tab[w][s] = f(16 w - 1, s), s < 16 w
  const int N = a.N, V = a.V, Np = (N + 15) & ~15, ldn = Np + 8;
  bf16* bs = reinterpret_cast<bf16*>(raw);  // [CL][ldn]
  bf16* xs = bs + SSD_CL * ldn;             // [CL][ldv]
  bf16* sh = xs + SSD_CL * ldv;             // [Np][ldv]
  bf16* sl = sh + Np * ldv;                 // [Np][ldv]
  const int* c = a.ctab + 4 * blockIdx.x;
  const int row0 = c[0], len = c[1], h = blockIdx.y, g = h / (a.H / a.G);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, t2 = (lane & 3) * 2;
  const bf16* base = (const bf16*)a.xbc + (size_t)row0 * a.xbc_stride;
  const bf16* before = (const bf16*)a.before + ((size_t)blockIdx.x * a.H + h) * 2 * N * V;
  const RowCopy rb(Np >> 3, tid, TH), rv((min(64, V) + 15) / 16 * 2, tid, TH);
  stage<TH>(rb, bs, ldn, base + (size_t)a.H * V + (size_t)g * N, a.xbc_stride, SSD_CL, len, N, Np, vec);
  const int r0 = warp * 16;  // this lane's rows: r0 + gr and r0 + gr + 8
  uint32_t C[NK][4];
  {
    const bf16* cp = base + (size_t)a.H * V + (size_t)(a.G + g) * N;
#pragma unroll
    for (int k = 0; k < NK; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = r0 + gr + (e & 1) * 8, col = k * 16 + t2 + (e >> 1) * 8;
        C[k][e] = 0;
        if (row < len && col < N) {
          const bf16* p = cp + (size_t)row * a.xbc_stride + col;
          if (vec) {
            C[k][e] = *reinterpret_cast<const uint32_t*>(p);
          } else {
            __nv_bfloat162 v = __halves2bfloat162(p[0], col + 1 < N ? p[1] : __float2bfloat16_rn(0.f));
            C[k][e] = *reinterpret_cast<uint32_t*>(&v);
          }
        }
      }
  }
  for (int s = tid; s < SSD_CL; s += TH) {
    float4 d = make_float4(0.f, 0.f, 0.f, 0.f);
    if (s < len) {
      const float4* dp = a.dec + (size_t)h * a.tokens + row0;
      d = dp[s];
      if (s >= SW_L) {  // the sums start over after 64 tokens
        float4 o = dp[SW_L - 1];
        float2 t = pair_add(make_float2(o.x, o.y), make_float2(d.x, d.y));
        d.x = t.x;
        d.y = t.y;
      }
    }
    cum[s] = make_float2(d.x, d.y);
    dts[s] = d.z;
  }
  const float skip = a.d[h];
  const int sv = (lane & 15) * ldv + (lane >> 4) * 8;
  for (int v0 = 0; v0 < V; v0 += 64) {
    const int cols = min(64, V - v0), colsp = (cols + 15) & ~15, nv = colsp >> 4;
    if (v0) __syncthreads();  // the tile before is done with xs, sh, sl
    stage<TH>(rv, xs, ldv, base + (size_t)h * V + v0, a.xbc_stride, SSD_CL, len, cols, colsp, vec);
    stage<TH>(rv, sh, ldv, before + v0, V, Np, N, cols, colsp, vec);
    stage<TH>(rv, sl, ldv, before + (size_t)N * V + v0, V, Np, N, cols, colsp, vec);
    cp_commit();
    if (v0 == 0) {
      __syncthreads();  // cum and dts are written
      for (int i = tid; i < SSD_CL / 16 * SSD_CL; i += TH) {
        const int w = i / SSD_CL, s = i % SSD_CL;
        if (s < 16 * w) tab[w][s] = dts[s] * expf(pair_diff(cum[16 * w - 1], cum[s]));
      }
    }
    cp_wait<0>();
    __syncthreads();
    if (r0 < len) {
      float acc[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        if (k * 16 >= Np) break;
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (i < nv) {
            uint32_t b[4], d[4];
            ldm4t(b, sh + k * 16 * ldv + sv + i * 16);
            ldm4t(d, sl + k * 16 * ldv + sv + i * 16);
            mma(acc[2 * i], C[k], b);
            mma(acc[2 * i + 1], C[k], b + 2);
            mma(acc[2 * i], C[k], d);
            mma(acc[2 * i + 1], C[k], d + 2);
          }
      }
      const float2 ct[2] = {cum[r0 + gr], cum[r0 + gr + 8]};
      float2 cr = make_float2(0.f, 0.f);
      if (warp) cr = cum[r0 - 1];
      const float er = expf(cr.x + cr.y);
#pragma unroll
      for (int i = 0; i < 8; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[i][e] *= er;
      for (int s0 = 0; s0 <= r0; s0 += 16) {
        float s[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
        const bf16* bp = bs + (s0 + (lane & 7) + (lane >> 4) * 8) * ldn + ((lane >> 3) & 1) * 8;
#pragma unroll
        for (int k = 0; k < NK; ++k) {
          if (k * 16 >= Np) break;
          uint32_t b[4];
          ldm4(b, bp + k * 16);
          mma(s[0], C[k], b);
          mma(s[1], C[k], b + 2);
        }
        if (s0 < r0) {
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const float2 f = *reinterpret_cast<const float2*>(&tab[warp][s0 + u * 8 + t2]);
            s[u][0] *= f.x; s[u][1] *= f.y; s[u][2] *= f.x; s[u][3] *= f.y;
          }
        } else {  // the rows' own tokens: everything so far belongs to tokens up to r
          const float e0 = expf(pair_diff(ct[0], cr)), e1 = expf(pair_diff(ct[1], cr));
#pragma unroll
          for (int i = 0; i < 8; ++i) { acc[i][0] *= e0; acc[i][1] *= e0; acc[i][2] *= e1; acc[i][3] *= e1; }
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const int src = s0 + u * 8 + t2;
            const float2 cs[2] = {cum[src], cum[src + 1]};
            const float w[2] = {dts[src], dts[src + 1]};
#pragma unroll
            for (int e = 0; e < 4; ++e)
              s[u][e] = src + (e & 1) <= r0 + gr + (e >> 1) * 8 ? s[u][e] * (w[e & 1] * expf(pair_diff(ct[e >> 1], cs[e & 1]))) : 0.f;
          }
        }
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          split2(s[u][0], s[u][1], hi[2 * u], lo[2 * u]);
          split2(s[u][2], s[u][3], hi[2 * u + 1], lo[2 * u + 1]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (i < nv) {
            uint32_t b[4];
            ldm4t(b, xs + s0 * ldv + sv + i * 16);
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
      f[e] *= silu_as<T>(g[e]);
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

// The chunked form (bf16), three launches.  -3: more than 256 state rows.
int hyb_ssd_chunked(const SsdArgs* args, cudaStream_t st) {
  const SsdArgs& a = *args;
  if (a.nseq == 0) return 0;
  if (a.G < 1 || a.H % a.G || a.N < 1 || a.V < 1) return -2;
  if (a.N > 256 || a.H > 65535) return -3;
  const size_t Np = (size_t)((a.N + 15) & ~15);
  const size_t sw = (SW_STAGES * SW_L * (Np + 8 + SW_VT + 8) + 4 * SW_L * (SW_VT + 8)) * sizeof(bf16);
  const size_t so = (SSD_CL * (Np + 8) + SSD_CL * 72 + 2 * Np * 72) * sizeof(bf16);
  const uintptr_t bits = (uintptr_t)a.xbc | (uintptr_t)a.y | (uintptr_t)a.before | (uintptr_t)a.dec;
  const int vec = (bits & 15) == 0 && ((a.N | a.V) & 7) == 0 && (a.xbc_stride & 7) == 0;
  dim3 wgrid(a.nseq, a.H, (a.V + SW_VT - 1) / SW_VT), ogrid(a.nchunks, a.H);
#define CK(MT, NK)                                                                                          \
  do {                                                                                                      \
    cudaFuncSetAttribute(ssd_walk_kernel<MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sw);        \
    cudaFuncSetAttribute(ssd_out_kernel<NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)so);         \
    ssd_decay_kernel<<<dim3(a.nchunks, (a.H + 3) / 4), 256, 0, st>>>(a);                                    \
    ssd_walk_kernel<MT><<<wgrid, SW_TH, sw, st>>>(a, vec);                                                  \
    ssd_out_kernel<NK><<<ogrid, 2 * SSD_CL, so, st>>>(a, vec);                                              \
  } while (0)
  if (a.N <= 64) CK(1, 4); else if (a.N <= 128) CK(1, 8); else CK(2, 16);
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

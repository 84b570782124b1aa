// Row kernels of the hybrid model family that join several steps of a block: the residual update of a sublayer with
// the average over depth and the next sublayer's input behind it, the norm with a short causal convolution over time,
// and the polynomial activation with its own norms.  Same conventions as hybrid_mixers.cu: a packed batch of N tokens,
// `meta[4*s] = {first token row, token count, slot, position of the first token}`, `tok_seq[i]` = sequence of row i,
// fp32 arithmetic whatever the activation type T (bf16 or fp32).
#include "hybrid_common.cuh"

namespace hyb {

#define HR_THREADS 256

// VEC neighbouring values (VEC = 4: one 16-byte access of fp32, one 8-byte access of bf16; VEC = 1: any width)
template <int VEC> __device__ __forceinline__ void ldv(const float* p, float* f) {
  if (VEC == 4) {
    float4 a = *reinterpret_cast<const float4*>(p);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  } else {
    f[0] = p[0];
  }
}
template <int VEC> __device__ __forceinline__ void ldv(const bf16* p, float* f) {
  if (VEC == 4) {
    uint2 u = *reinterpret_cast<const uint2*>(p);
    f[0] = __uint_as_float(u.x << 16); f[1] = __uint_as_float(u.x & 0xffff0000u);
    f[2] = __uint_as_float(u.y << 16); f[3] = __uint_as_float(u.y & 0xffff0000u);
  } else {
    f[0] = to_f(p[0]);
  }
}
template <int VEC> __device__ __forceinline__ void stv(float* p, const float* f) {
  if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  else p[0] = f[0];
}
template <int VEC> __device__ __forceinline__ void stv(bf16* p, const float* f) {
  if (VEC == 4) {
    __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
  } else {
    p[0] = __float2bfloat16_rn(f[0]);
  }
}

// Statistics of the row `buf[0..C)` in shared memory, each thread reading only the values it owns.
// kind 0: layer norm (mean and 1/sqrt(var + eps)); kind 1: RMS norm (mean = 0).  `s` is the thread's partial sum.
template <int VEC>
__device__ __forceinline__ void row_stats(const float* buf, int C, int kind, float eps, float s, float* red, float& mean, float& inv) {
  mean = 0.f;
  if (kind == 0) mean = block_sum(s, red) / C;
  float ss = 0.f;
  for (int c = threadIdx.x * VEC; c < C; c += HR_THREADS * VEC) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      float d = buf[c + e] - mean;
      ss += d * d;
    }
  }
  inv = 1.f / sqrtf(block_sum(ss, red) / C + eps);
}

// One row of a block's bookkeeping, one thread block per token row:
//   x   += mult * norm1(y)                                   (y == null: x stays as it is)
//   copy = x rounded to T                                    (copy != null)
//   avg  = sum_{j < n_avg} avg_w[j] * hist[j] + avg_w[n_avg] * x   (avg_out != null; hist rows are N*C apart)
//   h    = norm2(avg or x), then h + conv(h) over time       (w2 != null; steps of one token per sequence only)
// The convolution's earlier inputs come from conv_state[slot] ([taps-1, C] fp32, oldest first), which is advanced;
// positions before the sequence's start count as zero whatever the slot holds.
struct RowUpdateArgs {
  const void *y, *w1, *b1;
  float* x;
  void* copy;
  const float *hist, *avg_w;
  float* avg_out;
  const void *w2, *b2;
  const float* conv_w;   // [taps, C]: row taps-1 weighs the current token
  float* conv_state;
  void* h;
  const int *meta, *tok_seq;
  long long y_stride;
  int N, C, kind1, kind2, n_avg, taps;
  float eps1, eps2, mult;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(HR_THREADS) row_update_kernel(RowUpdateArgs a) {
  extern __shared__ float buf[];  // [C]
  __shared__ float red[33];
  const int C = a.C;
  const size_t row = (size_t)blockIdx.x * C;
  float* x = a.x + row;
  float mean, inv, s = 0.f;
  if (a.y) {
    const T* y = (const T*)a.y + (size_t)blockIdx.x * a.y_stride;
    for (int c = threadIdx.x * VEC; c < C; c += HR_THREADS * VEC) {
      float f[VEC];
      ldv<VEC>(y + c, f);
#pragma unroll
      for (int e = 0; e < VEC; ++e) { s += f[e]; buf[c + e] = f[e]; }
    }
    row_stats<VEC>(buf, C, a.kind1, a.eps1, s, red, mean, inv);
  }
  s = 0.f;
  for (int c = threadIdx.x * VEC; c < C; c += HR_THREADS * VEC) {
    float v[VEC];
    ldv<VEC>(x + c, v);
    if (a.y) {
      float w[VEC];
      ldv<VEC>((const T*)a.w1 + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) w[e] *= (buf[c + e] - mean) * inv;
      if (a.b1) {
        float b[VEC];
        ldv<VEC>((const T*)a.b1 + c, b);
#pragma unroll
        for (int e = 0; e < VEC; ++e) w[e] += b[e];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] += a.mult * w[e];
      stv<VEC>(x + c, v);
    }
    if (a.copy) stv<VEC>((T*)a.copy + row + c, v);
    if (a.avg_out) {
      const float wl = a.avg_w[a.n_avg];
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
      const float* hp = a.hist + row + c;
#pragma unroll 4
      for (int j = 0; j < a.n_avg; ++j) {
        float f[VEC];
        ldv<VEC>(hp + (size_t)j * a.N * C, f);
        const float wj = a.avg_w[j];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] += wj * f[e];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) v[e] = acc[e] + wl * v[e];
      stv<VEC>(a.avg_out + row + c, v);
    }
    if (a.w2) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) { s += v[e]; buf[c + e] = v[e]; }
    }
  }
  if (!a.w2) return;
  row_stats<VEC>(buf, C, a.kind2, a.eps2, s, red, mean, inv);
  const int* m = a.meta + 4 * a.tok_seq[blockIdx.x];
  const int taps = a.conv_w ? a.taps : 1, pos = m[3];
  float* st = a.conv_state ? a.conv_state + (size_t)m[2] * (taps - 1) * C : nullptr;
  for (int c = threadIdx.x * VEC; c < C; c += HR_THREADS * VEC) {
    float h[VEC], w[VEC], o[VEC];
    ldv<VEC>((const T*)a.w2 + c, w);
#pragma unroll
    for (int e = 0; e < VEC; ++e) h[e] = (buf[c + e] - mean) * inv * w[e];
    if (a.b2) {
      ldv<VEC>((const T*)a.b2 + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) h[e] += w[e];
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = h[e];
    if (a.conv_w) {
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
      for (int r = 0; r < taps - 1; ++r) {  // state row r: position pos - (taps - 1 - r)
        float f[VEC];
        ldv<VEC>(a.conv_w + (size_t)r * C + c, w);
        ldv<VEC>(st + (size_t)r * C + c, f);
        const bool before = pos - (taps - 1 - r) < 0;
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] += before ? 0.f : w[e] * f[e];
        if (r) stv<VEC>(st + (size_t)(r - 1) * C + c, f);
      }
      ldv<VEC>(a.conv_w + (size_t)(taps - 1) * C + c, w);
#pragma unroll
      for (int e = 0; e < VEC; ++e) o[e] = h[e] + (acc[e] + w[e] * h[e]);
      if (taps > 1) stv<VEC>(st + (size_t)(taps - 2) * C + c, h);
    }
    stv<VEC>((T*)a.h + row + c, o);
  }
}

// h = norm(x), out = h + conv(h) for steps that bring several tokens of a sequence.  A block owns `tile` consecutive token
// rows.  First its warps take the statistics of those rows and of the taps - 1 rows before them, one row per warp; then
// every thread walks its channels: a tap reads the earlier row again (it is in the first-level cache) and norms it on the
// fly, rows of earlier steps come from conv_state.  Blocks are independent.
// mode 0: outputs only.  mode 1: outputs, and the block that holds a sequence's last token writes its conv_state (allowed
// when no sequence of the step reads it: they all start at position 0).  mode 2: conv_state only, one block per sequence.
template <typename T, int VEC>
__global__ void __launch_bounds__(HR_THREADS) norm_conv_kernel(const float* __restrict__ x, const T* __restrict__ w,
                                                               const T* __restrict__ b, const float* __restrict__ conv_w,
                                                               float* __restrict__ state, T* __restrict__ out,
                                                               const int* __restrict__ meta, const int* __restrict__ tok_seq,
                                                               int N, int C, int taps, int kind, float eps, int tile, int mode) {
  extern __shared__ float2 stats[];  // (mean, 1 / deviation) of rows r0 .. last - 1
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int first = blockIdx.x * tile, last = min(N, first + tile);
  if (mode == 2) {
    const int* m = meta + 4 * blockIdx.x;
    last = m[0] + m[1];
    first = last;
  }
  const int r0 = max(0, first - (taps - 1));
  for (int r = r0 + warp; r < last; r += HR_THREADS / 32) {
    const float* row = x + (size_t)r * C;
    float mean = 0.f, s = 0.f, ss = 0.f;
    if (kind == 0) {
#pragma unroll 8
      for (int c = lane * VEC; c < C; c += 32 * VEC) {
        float f[VEC];
        ldv<VEC>(row + c, f);
#pragma unroll
        for (int e = 0; e < VEC; ++e) s += f[e];
      }
      mean = warp_sum(s) / C;
    }
#pragma unroll 8
    for (int c = lane * VEC; c < C; c += 32 * VEC) {
      float f[VEC];
      ldv<VEC>(row + c, f);
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss += (f[e] - mean) * (f[e] - mean);
    }
    ss = warp_sum(ss);
    if (lane == 0) stats[r - r0] = make_float2(mean, 1.f / sqrtf(ss / C + eps));
  }
  __syncthreads();
  auto normed = [&](int r, int c, const float* wv, const float* bv, float* o) {
    float2 t = stats[r - r0];
    ldv<VEC>(x + (size_t)r * C + c, o);
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = (o[e] - t.x) * t.y * wv[e] + bv[e];
  };
  for (int c = threadIdx.x * VEC; c < C; c += HR_THREADS * VEC) {
    float wv[VEC], bv[VEC];
    ldv<VEC>(w + c, wv);
    if (b) ldv<VEC>(b + c, bv);
    else
#pragma unroll
      for (int e = 0; e < VEC; ++e) bv[e] = 0.f;
    // the state rows of a sequence after its token `tok` (the last one): ascending, so an old row moves down in place
    auto advance = [&](const int* m, int tok) {
      float* st = state + (size_t)m[2] * (taps - 1) * C + c;
      for (int r = 0; r < taps - 1; ++r) {
        int local = tok - m[0] - (taps - 2 - r);
        float f[VEC];
        if (local >= 0) {
          normed(m[0] + local, c, wv, bv, f);
        } else if (m[3] + local < 0) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) f[e] = 0.f;
        } else {
          ldv<VEC>(st + (size_t)(r + m[1]) * C, f);
        }
        stv<VEC>(st + (size_t)r * C, f);
      }
    };
    if (mode == 2) {
      advance(meta + 4 * blockIdx.x, last - 1);
      continue;
    }
    for (int tok = first; tok < last; ++tok) {
      const int* m = meta + 4 * tok_seq[tok];
      const int local = tok - m[0];
      float acc[VEC], h[VEC], f[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
      for (int j = 0; j < taps; ++j) {
        const int src = local - (taps - 1 - j);
        if (src >= 0) {
          normed(m[0] + src, c, wv, bv, h);
        } else if (m[3] + src >= 0) {
          ldv<VEC>(state + ((size_t)m[2] * (taps - 1) + (taps - 1 + src)) * C + c, h);
        } else {
          continue;  // before the sequence's start, whatever the slot holds
        }
        ldv<VEC>(conv_w + (size_t)j * C + c, f);
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] += f[e] * h[e];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] += h[e];  // the last tap read the row itself
      stv<VEC>(out + (size_t)tok * C + c, acc);
      if (mode == 1 && local == m[1] - 1) advance(m, tok);
    }
  }
}

// z -> a N(z) + b N(z^2) + c N(z^3) + e, powers taken entry by entry, N(v) = v / sqrt(mean(v^2) + eps) over the row.
// One block per row, as many threads as the row fills with 8 values each (at most 1024); the three sums of squares are
// reduced together.  Rows of up to PN_KEEP * 8 values per thread stay in registers between the sums and the result.
#define PN_KEEP 2
template <typename T, bool VEC8>
__global__ void __launch_bounds__(1024) poly_norm_kernel(const T* z, long long z_stride, T* out, long long out_stride,
                                                         const float* __restrict__ coef, int F, float eps) {
  __shared__ float red[3][32];
  const T* src = z + (size_t)blockIdx.x * z_stride;
  T* dst = out + (size_t)blockIdx.x * out_stride;
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  float keep[VEC8 ? PN_KEEP : 1][8];
  auto add = [&](float v) {
    float v2 = v * v;
    s1 += v2;
    s2 += v2 * v2;
    s3 += (v2 * v) * (v2 * v);
  };
  if (VEC8) {
#pragma unroll
    for (int k = 0; k < PN_KEEP; ++k) {
      int c = (threadIdx.x + k * blockDim.x) * 8;
      if (c < F) load8(src + c, keep[k]);
    }
#pragma unroll
    for (int k = 0; k < PN_KEEP; ++k)
      if ((threadIdx.x + k * blockDim.x) * 8 < F)
#pragma unroll
        for (int e = 0; e < 8; ++e) add(keep[k][e]);
  } else {
    for (int c = threadIdx.x; c < F; c += blockDim.x) add(to_f(src[c]));
  }
  s1 = warp_sum(s1);
  s2 = warp_sum(s2);
  s3 = warp_sum(s3);
  const int lane = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  if (lane == 0) {
    red[0][threadIdx.x >> 5] = s1;
    red[1][threadIdx.x >> 5] = s2;
    red[2][threadIdx.x >> 5] = s3;
  }
  __syncthreads();
  s1 = warp_sum(lane < nw ? red[0][lane] : 0.f);
  s2 = warp_sum(lane < nw ? red[1][lane] : 0.f);
  s3 = warp_sum(lane < nw ? red[2][lane] : 0.f);
  const float a = coef[0] / sqrtf(s1 / F + eps), b = coef[1] / sqrtf(s2 / F + eps), c3 = coef[2] / sqrtf(s3 / F + eps), e0 = coef[3];
  if (VEC8) {
#pragma unroll
    for (int k = 0; k < PN_KEEP; ++k) {
      int c = (threadIdx.x + k * blockDim.x) * 8;
      if (c < F) {
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          float v = keep[k][e], v2 = v * v;
          keep[k][e] = a * v + b * v2 + c3 * (v2 * v) + e0;
        }
        store8(dst + c, keep[k]);
      }
    }
  } else {
    for (int c = threadIdx.x; c < F; c += blockDim.x) {
      float v = to_f(src[c]), v2 = v * v;
      dst[c] = from_f<T>(a * v + b * v2 + c3 * (v2 * v) + e0);
    }
  }
}

// One thread per sequence that brings several tokens: prev[slot] = its last token of the step.
__global__ void remember_tokens_kernel(const int* __restrict__ tokens, const int* __restrict__ meta, int nseq, int* __restrict__ prev) {
  int s = blockIdx.x * blockDim.x + threadIdx.x;
  if (s < nseq && meta[4 * s + 1] > 1) prev[meta[4 * s + 2]] = tokens[meta[4 * s] + meta[4 * s + 1] - 1];
}

// x = scale * table[token] + pair_table[row of (previous token, token)], row = (previous * mul_prev + token * mul_cur)
// mod buckets; a sequence's first token takes row `buckets`.  The token before a step's first one is prev[slot]; a
// sequence that brings one token leaves it there (longer ones: remember_tokens_kernel).  out2: a second copy of the row.
template <typename T, int VEC>
__global__ void embed_pairs_kernel(const T* __restrict__ table, const T* __restrict__ pair_table, const int* __restrict__ tokens,
                                   float* __restrict__ out, float* __restrict__ out2, int C, float scale, long long buckets,
                                   long long mul_prev, long long mul_cur, int* __restrict__ prev,
                                   const int* __restrict__ meta, const int* __restrict__ tok_seq) {
  __shared__ long long s_row;
  int t = blockIdx.x, tok = tokens[t];
  if (threadIdx.x == 0) {
    const int* m = meta + 4 * tok_seq[t];
    int local = t - m[0];
    long long r = buckets;
    if (m[3] + local > 0) {
      long long before = local > 0 ? tokens[t - 1] : prev[m[2]];
      r = (before * mul_prev + (long long)tok * mul_cur) % buckets;
      if (r < 0) r += buckets;
    }
    if (m[1] == 1) prev[m[2]] = tok;
    s_row = r;
  }
  __syncthreads();
  const T *src = table + (size_t)tok * C, *pr = pair_table + (size_t)s_row * C;
  for (int c = threadIdx.x * VEC; c < C; c += blockDim.x * VEC) {
    float f[VEC], g[VEC];
    ldv<VEC>(src + c, f);
    ldv<VEC>(pr + c, g);
#pragma unroll
    for (int e = 0; e < VEC; ++e) f[e] = scale * f[e] + g[e];
    stv<VEC>(out + (size_t)t * C + c, f);
    if (out2) stv<VEC>(out2 + (size_t)t * C + c, f);
  }
}

}  // namespace hyb

using namespace hyb;

static inline bool al16(const void* p) { return ((uintptr_t)p & 15) == 0; }

extern "C" {

int hyb_row_update(const RowUpdateArgs* args, int dt, cudaStream_t st) {
  const RowUpdateArgs& a = *args;
  if (a.N == 0) return 0;
  if (a.C < 1 || !a.x || (a.w2 && (!a.h || !a.meta || !a.tok_seq)) || (a.avg_out && (!a.hist || !a.avg_w))) return -2;
  if (a.w2 && a.conv_w && (a.taps < 1 || (a.taps > 1 && !a.conv_state))) return -2;
  size_t smem = (size_t)a.C * sizeof(float);
  if (smem > 200 * 1024) return -3;
  const void* ps[] = {a.y, a.w1, a.b1, a.x, a.copy, a.hist, a.avg_out, a.w2, a.b2, a.conv_w, a.conv_state, a.h};
  bool vec = a.C % 4 == 0 && a.y_stride % 4 == 0;
  for (const void* p : ps) vec = vec && al16(p);
#define RU(T, V)                                                                                            \
  do {                                                                                                      \
    if (smem > 40 * 1024)                                                                                   \
      cudaFuncSetAttribute(row_update_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    row_update_kernel<T, V><<<a.N, HR_THREADS, smem, st>>>(a);                                              \
  } while (0)
  if (dt == 0) { if (vec) RU(bf16, 4); else RU(bf16, 1); }
  else { if (vec) RU(float, 4); else RU(float, 1); }
#undef RU
  return (int)cudaGetLastError();
}

// carries != 0: some sequence of the step reads its conv_state (it does not start at position 0)
int hyb_norm_conv(const float* x, const void* w, const void* b, const float* conv_w, float* state, void* out, const int* meta,
                  const int* tok_seq, int N, int nseq, int C, int taps, int kind, float eps, int tile, int carries, int dt,
                  cudaStream_t st) {
  if (N == 0) return 0;
  if (taps < 1 || tile < 1 || C < 1 || (taps > 1 && !state)) return -2;
  size_t smem = (size_t)(tile + taps) * sizeof(float2);
  if (smem > 40 * 1024) return -3;
  bool vec = C % 4 == 0 && al16(x) && al16(w) && al16(b) && al16(conv_w) && al16(state) && al16(out);
  int blocks = (N + tile - 1) / tile, mode = taps > 1 && !carries ? 1 : 0;
#define NC(T, V)                                                                                                           \
  do {                                                                                                                     \
    norm_conv_kernel<T, V><<<blocks, HR_THREADS, smem, st>>>(x, (const T*)w, (const T*)b, conv_w, state, (T*)out, meta,    \
                                                             tok_seq, N, C, taps, kind, eps, tile, mode);                  \
    if (taps > 1 && carries)                                                                                               \
      norm_conv_kernel<T, V><<<nseq, HR_THREADS, smem, st>>>(x, (const T*)w, (const T*)b, conv_w, state, (T*)out, meta,    \
                                                             tok_seq, N, C, taps, kind, eps, tile, 2);                     \
  } while (0)
  if (dt == 0) { if (vec) NC(bf16, 4); else NC(bf16, 1); }
  else { if (vec) NC(float, 4); else NC(float, 1); }
#undef NC
  return (int)cudaGetLastError();
}

int hyb_poly_norm(const void* z, long long z_stride, void* out, long long out_stride, const float* coef, int rows, int F, float eps,
                  int dt, cudaStream_t st) {
  if (rows == 0) return 0;
  if (F < 1) return -2;
  bool vec = F % 8 == 0 && F <= PN_KEEP * 8 * 1024 && z_stride % 8 == 0 && out_stride % 8 == 0 && al16(z) && al16(out);
  int per = vec ? F / 8 : F, th = per >= 1024 ? 1024 : (per + 31) / 32 * 32;
  if (vec && th > 256 && rows >= 1184) th = ((per + PN_KEEP - 1) / PN_KEEP + 31) / 32 * 32;  // many rows: fewer, busier warps per row
#define PN(T, V) poly_norm_kernel<T, V><<<rows, th, 0, st>>>((const T*)z, z_stride, (T*)out, out_stride, coef, F, eps)
  if (dt == 0) { if (vec) PN(bf16, true); else PN(bf16, false); }
  else { if (vec) PN(float, true); else PN(float, false); }
#undef PN
  return (int)cudaGetLastError();
}

int hyb_embed_pairs(const void* table, const void* pair_table, const int* tokens, float* out, float* out2, int N, int nseq, int C,
                    float scale, long long buckets, long long mul_prev, long long mul_cur, int* prev, const int* meta,
                    const int* tok_seq, int several, int dt, cudaStream_t st) {
  if (N == 0) return 0;
  if (buckets < 1 || C < 1) return -2;
  bool vec = C % 4 == 0 && al16(table) && al16(pair_table) && al16(out) && al16(out2);
#define EP(T, V)                                                                                                     \
  embed_pairs_kernel<T, V><<<N, HR_THREADS, 0, st>>>((const T*)table, (const T*)pair_table, tokens, out, out2, C, scale, \
                                                     buckets, mul_prev, mul_cur, prev, meta, tok_seq)
  if (dt == 0) { if (vec) EP(bf16, 4); else EP(bf16, 1); }
  else { if (vec) EP(float, 4); else EP(float, 1); }
#undef EP
  if (several) remember_tokens_kernel<<<(nseq + 127) / 128, 128, 0, st>>>(tokens, meta, nseq, prev);
  return (int)cudaGetLastError();
}

}  // extern "C"

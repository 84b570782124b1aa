// Tensor-core forms of latent attention with 16-bit activations (the fp32 mode and shapes outside the stated multiples use
// the kernels of hybrid_mixers.cu and library matrix products):
//
//  * latent_decode_mma_kernel: one-token steps and short portions, straight on the cached rows [L latent | R rotated key].
//    All heads read the same rows, so 16 heads of a token are the rows of one matrix-product tile.
//  * prompt_attn_mma_kernel: prompts, on keys and values expanded per head, scores and weights never leave the SM.
//
// In both, a learned score per head (`sink`) may join the softmax denominator without a key or a value.
//
// Queries of the first kernel and softmax weights of both enter the products as a bf16 number plus the bf16 remainder, so
// they keep twice the mantissa; sums are fp32.  Warp-level m16n8k16 products: the tiles are 16 and 64 rows high and a
// step is bound by reading the cache (first kernel) or by its many small dependent tiles (second), see the bounds there.
#include "hybrid_mma.cuh"

namespace hyb {

// Block = one token x 16 heads x one share of its keys, 4 warps.  Tiles of 32 cached rows arrive by asynchronous 16-byte
// copies, two buffers.  Per tile: warp w computes the scores of keys 8w .. 8w+7 for the 16 heads (queries as hi + lo),
// then the softmax of heads 4w .. 4w+3 (lane = key), then the weighted sum for its quarter of the latent.
// Needs L + R a multiple of 16, L a multiple of 32 and at most 32 * NT (NT: 8-column tiles of a warp's quarter).
#define LD_TILE 32
template <int NT>
__global__ void __launch_bounds__(128) latent_decode_mma_kernel(const float* __restrict__ qlat, const bf16* __restrict__ q,
                                                                long long q_stride, const bf16* __restrict__ cache,
                                                                long long slot_stride, const int* __restrict__ meta,
                                                                const int* __restrict__ tok_seq, bf16* __restrict__ out, int N,
                                                                int H, int D, int R, int L, float scale, int nsplit,
                                                                float* __restrict__ part_acc, float* __restrict__ part_ml,
                                                                int window, const float* __restrict__ inv_freq, int nrot,
                                                                int interleaved, float amp, const float* __restrict__ sink) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float ss[16][LD_TILE + 1];
  __shared__ __align__(16) bf16 ph[16][LD_TILE + 8], pl[16][LD_TILE + 8];
  __shared__ float corr[16], fin[16];
  const int Dk = L + R, ld = Dk + 8;
  bf16* qh = reinterpret_cast<bf16*>(raw);        // [16][ld]
  bf16* ql = qh + 16 * ld;                        // [16][ld]
  bf16* kt = ql + 16 * ld;                        // [2][LD_TILE][ld]
  float2* cs = reinterpret_cast<float2*>(kt + 2 * LD_TILE * ld);  // [nrot / 2] (cos, sin) of the token's angles
  const int tok = blockIdx.x, h0 = blockIdx.y * 16, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int* m = meta + 4 * tok_seq[tok];
  const int pos = m[3] + tok - m[0], first = window > 0 ? max(0, pos - window + 1) : 0, nkeys = pos + 1 - first;
  const bf16* rows = cache + (size_t)m[2] * slot_stride + (size_t)first * Dk;
  const int chunk = ((nkeys + nsplit - 1) / nsplit + LD_TILE - 1) / LD_TILE * LD_TILE;
  const int k_begin = blockIdx.z * chunk, k_end = min(nkeys, k_begin + chunk);
  const int per = Dk >> 3;
  const RowCopy rc(per, tid, 128);
  auto fetch = [&](int t0, bf16* dst) {
    rc.run(dst, ld, rows + (size_t)t0 * Dk, Dk, LD_TILE, k_end - t0, Dk);
    cp_commit();
  };
  const bool any = k_begin < k_end;
  if (any) fetch(k_begin, kt);
  if (inv_freq)
    for (int i = tid; i < nrot / 2; i += 128) {
      float sn, co;
      sincosf((float)pos * inv_freq[i], &sn, &co);
      cs[i] = make_float2(co * amp, sn * amp);
    }
  __syncthreads();
  // queries to hi + lo; the loads of a thread are independent of one another, several in flight
  auto put = [&](int at, float v) {
    bf16 hi = __float2bfloat16_rn(v);
    qh[at] = hi;
    ql[at] = __float2bfloat16_rn(v - __bfloat162float(hi));
  };
  const int l4 = L >> 2;
#pragma unroll 8
  for (int i = tid; i < 16 * l4; i += 128) {
    int hh = i / l4, d = (i - hh * l4) * 4, h = h0 + hh;
    float4 v = *reinterpret_cast<const float4*>(qlat + ((size_t)min(h, H - 1) * N + tok) * L + d);
    float sc = h < H ? scale : 0.f;
    int at = hh * ld + d;
    put(at, v.x * sc);
    put(at + 1, v.y * sc);
    put(at + 2, v.z * sc);
    put(at + 3, v.w * sc);
  }
#pragma unroll 4
  for (int i = tid; i < 16 * R; i += 128) {
    int hh = i / R, r = i - hh * R, h = h0 + hh;
    const bf16* qr = q + (size_t)tok * q_stride + (size_t)min(h, H - 1) * (D + R) + D;
    const bool turn = inv_freq && r < nrot;
    const int half = nrot / 2, p = !turn ? 0 : interleaved ? r >> 1 : (r < half ? r : r - half);
    const int a = !turn ? r : interleaved ? 2 * p : p, b = !turn ? r : interleaved ? 2 * p + 1 : p + half;
    float va = to_f(qr[a]), vb = to_f(qr[b]);
    float2 t = turn ? cs[p] : make_float2(1.f, 0.f);
    put(hh * ld + L + r, (r == a ? va * t.x - vb * t.y : vb * t.x + va * t.y) * (h < H ? scale : 0.f));
  }
  float mx[4], l[4], acc[NT][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) { mx[i] = -INFINITY; l[i] = 0.f; }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  const int nt = L >> 5, col0 = warp * (L >> 2), g = lane >> 2, t2 = (lane & 3) * 2;
  int buf = 0;
  for (int t0 = k_begin; t0 < k_end; t0 += LD_TILE, buf ^= 1) {
    bf16* k = kt + buf * LD_TILE * ld;
    if (t0 + LD_TILE < k_end) { fetch(t0 + LD_TILE, kt + (buf ^ 1) * LD_TILE * ld); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    {
      float c0[4] = {0.f, 0.f, 0.f, 0.f}, c1[4] = {0.f, 0.f, 0.f, 0.f};
      const bf16* ap = qh + (lane & 15) * ld + (lane >> 4) * 8;
      const bf16* al = ql + (lane & 15) * ld + (lane >> 4) * 8;
      const bf16* bp = k + (warp * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8;
#pragma unroll 4
      for (int kk = 0; kk < Dk; kk += 16) {
        uint32_t a[4], b[2];
        ldm2(b, bp + kk);
        ldm4(a, ap + kk);
        mma(c0, a, b);
        ldm4(a, al + kk);
        mma(c1, a, b);
      }
      int c = warp * 8 + t2;
      ss[g][c] = c0[0] + c1[0];
      ss[g][c + 1] = c0[1] + c1[1];
      ss[g + 8][c] = c0[2] + c1[2];
      ss[g + 8][c + 1] = c0[3] + c1[3];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      int hh = warp * 4 + i;
      float s = t0 + lane < k_end ? ss[hh][lane] : -INFINITY;
      float mn = fmaxf(mx[i], warp_max(s));  // finite: a tile holds at least one key
      float cr = expf(mx[i] - mn), p = expf(s - mn);
      l[i] = l[i] * cr + warp_sum(p);
      mx[i] = mn;
      bf16 hi = __float2bfloat16_rn(p);
      ph[hh][lane] = hi;
      pl[hh][lane] = __float2bfloat16_rn(p - __bfloat162float(hi));
      if (lane == 0) corr[hh] = cr;
    }
    __syncthreads();
    {
      const float ca = corr[g], cb = corr[g + 8];
      uint32_t a[2][4], al[2][4];
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        ldm4(a[s], &ph[lane & 15][s * 16 + (lane >> 4) * 8]);
        ldm4(al[s], &pl[lane & 15][s * 16 + (lane >> 4) * 8]);
      }
#pragma unroll
      for (int i = 0; i < NT; ++i)
        if (i < nt) {
          acc[i][0] *= ca; acc[i][1] *= ca; acc[i][2] *= cb; acc[i][3] *= cb;
#pragma unroll
          for (int s = 0; s < 2; ++s) {
            uint32_t b[2];
            ldm2t(b, k + (s * 16 + (lane & 15)) * ld + col0 + i * 8);
            mma(acc[i], a[s], b);
            mma(acc[i], al[s], b);
          }
        }
    }
    __syncthreads();
  }
  if (lane == 0)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      int h = h0 + warp * 4 + i;
      float f = 1.f;
      if (nsplit == 1) {
        float sv = sink && h < H ? sink[h] : -INFINITY, M = fmaxf(mx[i], sv), e = expf(mx[i] - M);
        f = e / (l[i] * e + expf(sv - M));
      }
      fin[warp * 4 + i] = f;
      if (nsplit > 1 && h < H) {
        size_t b = ((size_t)blockIdx.z * H + h) * N + tok;
        part_ml[b * 2] = mx[i];
        part_ml[b * 2 + 1] = l[i];
      }
    }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < NT; ++i)
    if (i < nt) {
      int c = col0 + i * 8 + t2;
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        int hh = g + 8 * r, h = h0 + hh;
        if (h >= H) continue;
        float x = acc[i][2 * r] * fin[hh], y = acc[i][2 * r + 1] * fin[hh];
        if (nsplit == 1) *reinterpret_cast<__nv_bfloat162*>(out + ((size_t)h * N + tok) * L + c) = __floats2bfloat162_rn(x, y);
        else *reinterpret_cast<float2*>(part_acc + (((size_t)blockIdx.z * H + h) * N + tok) * L + c) = make_float2(x, y);
      }
    }
}

// Merge of the key shares: one warp per (token, head), nsplit <= 32.  Lane z reads share z's maximum and denominator, the
// weights e^(m_z - m) are handed round by shuffles while the lanes walk the latent four values at a time.
__global__ void latent_merge_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml, bf16* __restrict__ out,
                                    int N, int H, int L, int nsplit, const float* __restrict__ sink) {
  int tok = blockIdx.x, h = blockIdx.y, w = threadIdx.x >> 5, nw = blockDim.x >> 5, lane = threadIdx.x & 31;
  float ms = -INFINITY, ls = 0.f;
  if (lane < nsplit) {
    const float* ml = part_ml + (((size_t)lane * H + h) * N + tok) * 2;
    ms = ml[0];
    ls = ml[1];
  }
  const float sv = sink ? sink[h] : -INFINITY;
  float M = fmaxf(warp_max(ms), sv);
  float ws = lane < nsplit ? expf(ms - M) : 0.f;  // a share without keys: exp(-inf) = 0
  float inv = 1.f / (warp_sum(ls * ws) + expf(sv - M));
  for (int d0 = w * 128; d0 < L; d0 += nw * 128) {
    int d = d0 + 4 * lane;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int z = 0; z < nsplit; ++z) {
      float wz = __shfl_sync(0xffffffffu, ws, z);
      if (d < L) {
        float4 x = *reinterpret_cast<const float4*>(part_acc + (((size_t)z * H + h) * N + tok) * L + d);
        a.x += x.x * wz; a.y += x.y * wz; a.z += x.z * wz; a.w += x.w * wz;
      }
    }
    if (d < L) {
      __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(out + ((size_t)h * N + tok) * L + d);
      o[0] = __floats2bfloat162_rn(a.x * inv, a.y * inv);
      o[1] = __floats2bfloat162_rn(a.z * inv, a.w * inv);
    }
  }
}

// Prompt attention of all sequences of a step.  spans[5*z] = {first query row, n, first key row, p0, first}: sequence z has
// query rows i < n at positions p0 + i and the expanded keys of positions first .. p0 + n - 1, of which a row sees those not
// later than itself and (window > 0) fewer than `window` positions back.
// q rows: [H][DK] (rotated); kv rows: [G][DK] keys, then [G][V] values; out [n][H][V]; query head h reads head h / (H / G).
// sink (optional, fp32 [H]): one more score in a row's denominator.  gate (optional, [rows][H]): a head's
// output is multiplied by its sigmoid.
// Block = 64 query rows of one head, 4 warps of 16 rows; key tiles of PA_KEYS, two buffers, filled by asynchronous 16-byte
// copies while the tile before is used.  Scores and softmax weights stay in registers.  SPLIT: the weights enter the second
// product with their bf16 remainder.  Needs DK and V multiples of 16, V <= 8 NV.
#define PA_ROWS 64
template <int NV, int PA_KEYS, bool SPLIT>
__global__ void __launch_bounds__(128) prompt_attn_mma_kernel(const bf16* __restrict__ q, long long q_stride,
                                                              const bf16* __restrict__ kv, long long kv_stride,
                                                              bf16* __restrict__ out, const int* __restrict__ spans, int H,
                                                              int G, int DK, int V, int window, float scale_log2e,
                                                              const float* __restrict__ sink, const bf16* __restrict__ gate,
                                                              long long gate_stride) {
  const int* sp = spans + 5 * blockIdx.z;
  const int n = sp[1], p0 = sp[3], first = sp[4], keys = p0 + n - first;
  const int tiles = (n + PA_ROWS - 1) / PA_ROWS;
  if ((int)blockIdx.x >= tiles) return;
  q += (size_t)sp[0] * q_stride;
  kv += (size_t)sp[2] * kv_stride;
  out += (size_t)sp[0] * H * V;
  if (gate) gate += (size_t)sp[0] * gate_stride;
  extern __shared__ __align__(16) unsigned char raw[];
  const int ldk = DK + 8, ldv = V + 8;
  bf16* qs = reinterpret_cast<bf16*>(raw);     // [64][ldk]
  bf16* ks = qs + PA_ROWS * ldk;               // [2][64][ldk]
  bf16* vs = ks + 2 * PA_KEYS * ldk;           // [2][64][ldv]
  const int h = blockIdx.y, i0 = (tiles - 1 - (int)blockIdx.x) * PA_ROWS;  // long rows of work first
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
  const int dk8 = DK >> 3, v8 = V >> 3;
  const int kb = window > 0 ? max(0, p0 + i0 - window + 1 - first) : 0;
  const int ke = min(keys, p0 + min(n, i0 + PA_ROWS) - first);
  const int hk = h / (H / G);
  const bf16* kbase = kv + (size_t)hk * DK;
  const bf16* vbase = kv + (size_t)G * DK + (size_t)hk * V;
  const RowCopy rk(dk8, tid, 128), rv(v8, tid, 128);
  auto fetch = [&](int j0, int buf) {
    rk.run(ks + buf * PA_KEYS * ldk, ldk, kbase + (size_t)j0 * kv_stride, kv_stride, PA_KEYS, ke - j0, DK);
    rv.run(vs + buf * PA_KEYS * ldv, ldv, vbase + (size_t)j0 * kv_stride, kv_stride, PA_KEYS, ke - j0, V);
    cp_commit();
  };
  rk.run(qs, ldk, q + (size_t)i0 * q_stride + (size_t)h * DK, q_stride, PA_ROWS, n - i0, DK);
  fetch(kb, 0);  // kb < ke: row i0 sees at least itself
  float o[NV][4], mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
  const int nv2 = V >> 4;
  const int pr0 = p0 + i0 + warp * 16 + g - first;  // this lane's rows (pr0, pr0 + 8) as key indices
  int buf = 0;
  for (int j0 = kb; j0 < ke; j0 += PA_KEYS, buf ^= 1) {
    if (j0 + PA_KEYS < ke) { fetch(j0 + PA_KEYS, buf ^ 1); cp_wait<1>(); }
    else cp_wait<0>();
    __syncthreads();
    float s[PA_KEYS / 8][4];
#pragma unroll
    for (int i = 0; i < PA_KEYS / 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
    const bf16* ap = qs + (warp * 16 + (lane & 15)) * ldk + (lane >> 4) * 8;
    const bf16* bp = ks + (buf * PA_KEYS + (lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8;
#pragma unroll 2
    for (int kk = 0; kk < DK; kk += 16) {
      uint32_t a[4], b[4];
      ldm4(a, ap + kk);
#pragma unroll
      for (int i = 0; i < PA_KEYS / 16; ++i) {
        ldm4(b, bp + i * 16 * ldk + kk);
        mma(s[2 * i], a, b);
        mma(s[2 * i + 1], a, b + 2);
      }
    }
    float mn[2] = {mx[0], mx[1]};
    // tiles wholly inside every row's range need no mask
    const bool edge = j0 + PA_KEYS - 1 > p0 + i0 - first || (window > 0 && p0 + i0 + PA_ROWS - 1 - first - j0 >= window) || j0 + PA_KEYS > ke;
#pragma unroll
    for (int i = 0; i < PA_KEYS / 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = s[i][e] * scale_log2e;
        if (edge) {
          int j = j0 + i * 8 + t2 + (e & 1), p = pr0 + (e >> 1) * 8;
          if (j > p || j >= ke || (window > 0 && p - j >= window)) v = -INFINITY;
        }
        s[i][e] = v;
        mn[e >> 1] = fmaxf(mn[e >> 1], v);
      }
    float cr[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mn[r] = fmaxf(mn[r], __shfl_xor_sync(0xffffffffu, mn[r], 1));
      mn[r] = fmaxf(mn[r], __shfl_xor_sync(0xffffffffu, mn[r], 2));
      float safe = mn[r] == -INFINITY ? 0.f : mn[r];  // a row that has seen no key yet
      cr[r] = exp2f(mx[r] - safe);
      mx[r] = mn[r];
      mn[r] = safe;
      l[r] *= cr[r];
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) { o[i][0] *= cr[0]; o[i][1] *= cr[0]; o[i][2] *= cr[1]; o[i][3] *= cr[1]; }
    const bf16* vp = vs + (buf * PA_KEYS + (lane & 15)) * ldv + (lane >> 4) * 8;
#pragma unroll
    for (int kk = 0; kk < PA_KEYS / 16; ++kk) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        float* p = s[2 * kk + u];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          p[e] = exp2f(p[e] - mn[e >> 1]);
          l[e >> 1] += p[e];
        }
        split2(p[0], p[1], hi[2 * u], lo[2 * u]);
        split2(p[2], p[3], hi[2 * u + 1], lo[2 * u + 1]);
      }
#pragma unroll
      for (int i = 0; i < NV / 2; ++i)
        if (i < nv2) {
          uint32_t b[4];
          ldm4t(b, vp + kk * 16 * ldv + i * 16);
          mma(o[2 * i], hi, b);
          mma(o[2 * i + 1], hi, b + 2);
          if (SPLIT) {
            mma(o[2 * i], lo, b);
            mma(o[2 * i + 1], lo, b + 2);
          }
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    int row = i0 + warp * 16 + g + 8 * r;
    if (row >= n) continue;
    float inv;
    if (sink) {
      float sv = sink[h] * 1.4426950408889634f, M = fmaxf(mx[r], sv), e = exp2f(mx[r] - M);
      inv = e / (l[r] * e + exp2f(sv - M));
    } else {
      inv = 1.f / l[r];
    }
    if (gate) inv *= sigmoidf_(to_f(gate[(size_t)row * gate_stride + h]));
    bf16* dst = out + ((size_t)row * H + h) * V + t2;
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (i * 8 < V) *reinterpret_cast<__nv_bfloat162*>(dst + i * 8) = __floats2bfloat162_rn(o[i][2 * r] * inv, o[i][2 * r + 1] * inv);
  }
}

}  // namespace hyb

using namespace hyb;

extern "C" {

// -3: a shape or alignment these kernels do not take (the caller has another form)
int hyb_latent_decode_mma(const float* qlat, const void* q, long long q_stride, const void* cache, long long slot_stride,
                          const int* meta, const int* tok_seq, void* out, int N, int H, int D, int R, int L, float scale, int nsplit,
                          float* part_acc, float* part_ml, int window, const float* inv_freq, int nrot, int interleaved,
                          float amp, const float* sink, cudaStream_t st) {
  if (N == 0) return 0;
  if (nsplit < 1 || nsplit > 32 || (nsplit > 1 && (!part_acc || !part_ml)) || nrot > R || (nrot & 1)) return -2;
  int Dk = L + R;
  if (Dk % 16 || L % 32 || L > 512 || slot_stride % 8 || ((uintptr_t)cache & 15)) return -3;
  size_t smem = (size_t)(32 + 2 * LD_TILE) * (Dk + 8) * sizeof(bf16) + (size_t)(nrot / 2) * sizeof(float2);
  if (smem > 200 * 1024) return -3;
  dim3 grid(N, (H + 15) / 16, nsplit);
#define LM(NT)                                                                                                           \
  do {                                                                                                                   \
    cudaFuncSetAttribute(latent_decode_mma_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);          \
    latent_decode_mma_kernel<NT><<<grid, 128, smem, st>>>(qlat, (const bf16*)q, q_stride, (const bf16*)cache, slot_stride, \
                                                          meta, tok_seq, (bf16*)out, N, H, D, R, L, scale, nsplit, part_acc, \
                                                          part_ml, window, inv_freq, nrot, interleaved, amp, sink);      \
  } while (0)
  if (L <= 128) LM(4); else LM(16);
#undef LM
  if (nsplit > 1) latent_merge_kernel<<<dim3(N, H), L > 256 ? 128 : 64, 0, st>>>(part_acc, part_ml, (bf16*)out, N, H, L, nsplit, sink);
  return (int)cudaGetLastError();
}

int hyb_prompt_attn_mma(const void* q, long long q_stride, const void* kv, long long kv_stride, void* out, const int* spans,
                        int nseq, int longest, int H, int G, int DK, int V, int window, float scale, int split, int tile,
                        const float* sink, const void* gate, long long gate_stride, cudaStream_t st) {
  if (nseq == 0 || longest == 0) return 0;
  if ((tile != 32 && tile != 64) || G < 1 || H % G) return -2;
  uintptr_t bits = (uintptr_t)q | (uintptr_t)kv | (uintptr_t)out;
  if (DK % 16 || V % 16 || V > 256 || q_stride % 8 || kv_stride % 8 || (bits & 15) || scale <= 0.f) return -3;
  size_t smem = ((size_t)(PA_ROWS + 2 * tile) * (DK + 8) + (size_t)2 * tile * (V + 8)) * sizeof(bf16);
  if (smem > 200 * 1024) return -3;
  if (nseq > 65535 || H > 65535) return -3;
  dim3 grid((longest + PA_ROWS - 1) / PA_ROWS, H, nseq);
  const float sl = scale * 1.4426950408889634f;
#define PM(NV, KT, SP)                                                                                                    \
  do {                                                                                                                    \
    cudaFuncSetAttribute(prompt_attn_mma_kernel<NV, KT, SP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
    prompt_attn_mma_kernel<NV, KT, SP><<<grid, 128, smem, st>>>((const bf16*)q, q_stride, (const bf16*)kv, kv_stride,     \
                                                                (bf16*)out, spans, H, G, DK, V, window, sl, sink,         \
                                                                (const bf16*)gate, gate_stride);                          \
  } while (0)
#define PMT(NV) do { if (tile == 32) { if (split) PM(NV, 32, true); else PM(NV, 32, false); } \
                     else { if (split) PM(NV, 64, true); else PM(NV, 64, false); } } while (0)
  if (V <= 64) PMT(8); else if (V <= 128) PMT(16); else PMT(32);
#undef PMT
#undef PM
  return (int)cudaGetLastError();
}

}  // extern "C"

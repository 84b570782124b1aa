// Grouped-query attention of single tokens over cached rows [G * D keys | G * V values] with 16-bit activations, on the
// tensor cores: the query heads of a key/value head are the rows of a 16-row tile (hyb_window_attn in hybrid_mixers.cu is
// the form for fp32 and for sizes this one does not take; same masks, sinks, gates and soft cap).
//
// Block = (token, key/value head and 16 of its query heads, key share), 4 warps.  The warps walk 16-key tiles of the share in
// turn, each with its own ring of asynchronous copies, running maximum, denominator and sum, so the loop has no block
// barrier; their results meet in shared memory at the end.  Queries are bf16 as they come; softmax weights enter the
// second product as a bf16 number plus its bf16 remainder.
#include "hybrid_mma.cuh"

namespace hyb {

struct GroupedArgs {
  const bf16 *q, *gate, *cache;
  bf16* out;
  const int *meta, *tok_seq;
  const float* sink_vals;
  float *part_acc, *part_ml;
  long long q_stride, g_stride, slot_stride;
  int N, H, G, D, V, window, nsplit, mask_kind, sink, gate_mode;
  float scale, cap;
};

#define GD_KEYS 16
#define GD_STAGES 3
template <int NV>
__global__ void __launch_bounds__(128) grouped_decode_mma_kernel(GroupedArgs a) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float rm[4][16], rl[4][16];
  const int D = a.D, V = a.V, ldk = D + 8, ldv = V + 8, rep = a.H / a.G, tiles16 = (rep + 15) >> 4;
  const int t = blockIdx.x, g = blockIdx.y / tiles16, hb = (blockIdx.y - g * tiles16) * 16, live = min(16, rep - hb);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gr = lane >> 2, t2 = (lane & 3) * 2;
  bf16* qs = reinterpret_cast<bf16*>(raw);                                        // [16][ldk]
  bf16* ring = qs + 16 * ldk + warp * GD_STAGES * GD_KEYS * (ldk + ldv);           // [stages][keys][ldk], [keys][ldv]
  const int* m = a.meta + 4 * a.tok_seq[t];
  const int pos = m[3] + (t - m[0]);
  const int lo = a.window > 0 ? (a.mask_kind == 1 ? (pos / a.window) * a.window : max(0, pos - a.window + 1)) : 0;
  const int share = ((pos + 1 - lo + a.nsplit - 1) / a.nsplit + 63) & ~63;
  const int kb = lo + blockIdx.z * share, ke = min(pos + 1, kb + share);
  const size_t rowlen = (size_t)a.G * (D + V);
  const bf16* base = a.cache + (size_t)m[2] * a.slot_stride;
  const int dk8 = D >> 3;
  const RowCopy rk(dk8, lane, 32), rv(V >> 3, lane, 32);
  const int nt = kb < ke ? max(0, ((ke - kb + GD_KEYS - 1) / GD_KEYS - warp + 3) / 4) : 0;
  auto fetch = [&](int it) {
    if (it < nt) {
      bf16* k = ring + (it % GD_STAGES) * GD_KEYS * (ldk + ldv);
      bf16* v = k + GD_KEYS * ldk;
      const int j0 = kb + (warp + 4 * it) * GD_KEYS;
      const bf16* row = base + (size_t)j0 * rowlen;
      rk.run(k, ldk, row + (size_t)g * D, rowlen, GD_KEYS, ke - j0, D);
      rv.run(v, ldv, row + (size_t)a.G * D + (size_t)g * V, rowlen, GD_KEYS, ke - j0, V);
    }
    cp_commit();  // possibly an empty group: the wait counts groups
  };
#pragma unroll
  for (int i = 0; i < GD_STAGES - 1; ++i) fetch(i);
  for (int i = tid; i < 16 * dk8; i += 128) {
    int j = i / dk8, c = (i - j * dk8) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (j < live) v = *reinterpret_cast<const uint4*>(a.q + (size_t)t * a.q_stride + (size_t)(g * rep + hb + j) * D + c);
    *reinterpret_cast<uint4*>(qs + j * ldk + c) = v;
  }
  __syncthreads();
  float acc[NV][4], mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  const int nv2 = V >> 4;
  const bf16* ap = qs + (lane & 15) * ldk + (lane >> 4) * 8;
  for (int it = 0; it < nt; ++it) {
    cp_wait<GD_STAGES - 2>();
    __syncwarp();  // the tile has arrived for every lane, and every lane is done with the one the next fetch overwrites
    fetch(it + GD_STAGES - 1);
    const bf16* k = ring + (it % GD_STAGES) * GD_KEYS * (ldk + ldv);
    const bf16* v = k + GD_KEYS * ldk;
    float s[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[i][e] = 0.f;
    const bf16* bp = k + ((lane & 7) + (lane >> 4) * 8) * ldk + ((lane >> 3) & 1) * 8;
#pragma unroll 4
    for (int kk = 0; kk < D; kk += 16) {
      uint32_t A[4], b[4];
      ldm4(A, ap + kk);
      ldm4(b, bp + kk);
      mma(s[0], A, b);
      mma(s[1], A, b + 2);
    }
    const int j0 = kb + (warp + 4 * it) * GD_KEYS;
    float mn[2] = {mx[0], mx[1]};
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float x = s[u][e] * a.scale;
        if (a.cap > 0.f) x = a.cap * tanhf(x / a.cap);
        s[u][e] = j0 + u * 8 + t2 + (e & 1) < ke ? x : -INFINITY;
        mn[e >> 1] = fmaxf(mn[e >> 1], s[u][e]);
      }
    float cr[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {  // finite: a tile holds at least one key
      mn[r] = fmaxf(mn[r], __shfl_xor_sync(0xffffffffu, mn[r], 1));
      mn[r] = fmaxf(mn[r], __shfl_xor_sync(0xffffffffu, mn[r], 2));
      cr[r] = expf(mx[r] - mn[r]);
      mx[r] = mn[r];
      l[r] *= cr[r];
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) { acc[i][0] *= cr[0]; acc[i][1] *= cr[0]; acc[i][2] *= cr[1]; acc[i][3] *= cr[1]; }
    uint32_t hi[4], lw[4];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[u][e] = expf(s[u][e] - mn[e >> 1]);
        l[e >> 1] += s[u][e];
      }
      split2(s[u][0], s[u][1], hi[2 * u], lw[2 * u]);
      split2(s[u][2], s[u][3], hi[2 * u + 1], lw[2 * u + 1]);
    }
    const bf16* vp = v + (lane & 15) * ldv + (lane >> 4) * 8;
#pragma unroll
    for (int i = 0; i < NV / 2; ++i)
      if (i < nv2) {
        uint32_t b[4];
        ldm4t(b, vp + i * 16);
        mma(acc[2 * i], hi, b);
        mma(acc[2 * i + 1], hi, b + 2);
        mma(acc[2 * i], lw, b);
        mma(acc[2 * i + 1], lw, b + 2);
      }
    __syncwarp();
  }
  cp_wait<0>();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if ((lane & 3) == 0) { rm[warp][gr + 8 * r] = mx[r]; rl[warp][gr + 8 * r] = l[r]; }
  }
  __syncthreads();  // every warp is done with its ring
  float* ob = reinterpret_cast<float*>(raw);  // [4][16][V]
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = gr + 8 * r;
    if (row >= live) continue;
    const float M = fmaxf(fmaxf(rm[0][row], rm[1][row]), fmaxf(rm[2][row], rm[3][row]));
    const float w = M == -INFINITY ? 0.f : expf(mx[r] - M);
#pragma unroll
    for (int i = 0; i < NV; ++i)
      if (i * 8 < V) *reinterpret_cast<float2*>(ob + (warp * 16 + row) * V + i * 8 + t2) = make_float2(acc[i][2 * r] * w, acc[i][2 * r + 1] * w);
  }
  __syncthreads();
  for (int i = tid; i < live * V; i += 128) {
    const int row = i / V, d = i - row * V, h = g * rep + hb + row;
    float M = fmaxf(fmaxf(rm[0][row], rm[1][row]), fmaxf(rm[2][row], rm[3][row])), L = 0.f, o = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      L += M == -INFINITY ? 0.f : rl[w][row] * expf(rm[w][row] - M);
      o += ob[(w * 16 + row) * V + d];
    }
    if (a.nsplit > 1) {
      const size_t at = ((size_t)blockIdx.z * a.N + t) * a.H + h;
      a.part_acc[at * V + d] = o;
      if (d == 0) { a.part_ml[2 * at] = M; a.part_ml[2 * at + 1] = L; }
      continue;
    }
    if (a.sink) {  // the slot without a value
      const float sv = a.sink_vals ? a.sink_vals[h] : 0.f, Ms = fmaxf(M, sv), e = expf(M - Ms);
      L = L * e + expf(sv - Ms);
      o *= e;
    }
    o /= L;
    if (a.gate_mode == 1) o *= sigmoidf_(to_f(a.gate[(size_t)t * a.g_stride + h]));
    else if (a.gate_mode == 2) o *= sigmoidf_(to_f(a.gate[(size_t)t * a.g_stride + (size_t)h * V + d]));
    a.out[((size_t)t * a.H + h) * V + d] = __float2bfloat16_rn(o);
  }
}

}  // namespace hyb

using namespace hyb;

extern "C" {

// hybrid_mixers.cu: merges the key shares of single-token attention and applies sink and gate
int hyb_window_combine(const float* part_acc, const float* part_ml, const void* gate, long long g_stride, void* out, int N, int H, int V,
                       int nsplit, int sink, int gate_mode, const float* sink_vals, int dt, cudaStream_t st);

// -3: a shape or alignment this kernel does not take
int hyb_grouped_decode_mma(const void* q, long long q_stride, const void* gate, long long g_stride, const void* cache,
                           long long slot_stride, const int* meta, const int* tok_seq, void* out, int N, int H, int G, int D, int V,
                           float scale, int window, int nsplit, float* part_acc, float* part_ml, int mask_kind, int sink, int gate_mode,
                           float cap, const float* sink_vals, cudaStream_t st) {
  if (N == 0) return 0;
  if (G < 1 || H % G || nsplit < 1 || nsplit > 32 || (nsplit > 1 && (!part_acc || !part_ml)) || (gate_mode && !gate)) return -2;
  const int rep = H / G;
  const size_t smem = ((size_t)16 * (D + 8) + (size_t)4 * GD_STAGES * GD_KEYS * (D + V + 16)) * sizeof(bf16);
  if (D % 16 || V % 16 || D > 256 || V > 256 || q_stride % 8 || slot_stride % 8 || (((uintptr_t)q | (uintptr_t)cache) & 15) || smem > 220 * 1024) return -3;
  GroupedArgs a;
  a.q = (const bf16*)q; a.gate = (const bf16*)gate; a.cache = (const bf16*)cache; a.out = (bf16*)out; a.meta = meta; a.tok_seq = tok_seq;
  a.sink_vals = sink_vals; a.part_acc = part_acc; a.part_ml = part_ml; a.q_stride = q_stride; a.g_stride = g_stride; a.slot_stride = slot_stride;
  a.N = N; a.H = H; a.G = G; a.D = D; a.V = V; a.window = window; a.nsplit = nsplit; a.mask_kind = mask_kind; a.sink = sink;
  a.gate_mode = gate ? gate_mode : 0; a.scale = scale; a.cap = cap;
  dim3 grid(N, G * ((rep + 15) / 16), nsplit);
#define GD(NV)                                                                                                          \
  do {                                                                                                                  \
    cudaFuncSetAttribute(grouped_decode_mma_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);        \
    grouped_decode_mma_kernel<NV><<<grid, 128, smem, st>>>(a);                                                          \
  } while (0)
  if (V <= 64) GD(8); else if (V <= 128) GD(16); else GD(32);
#undef GD
  int rc = (int)cudaGetLastError();
  if (rc || nsplit == 1) return rc;
  return hyb_window_combine(part_acc, part_ml, gate, g_stride, out, N, H, V, nsplit, sink, a.gate_mode, sink_vals, 0, st);
}

}  // extern "C"

// Softmax attention over cached keys and values in a sliding window: groups of query heads share a key/value head, the first
// `keep` tokens stay visible, a sink may enter the denominator, a gate the result.  With two maps (differential attention)
// every head is two attentions over the same values, o = a1 - lambda a2, normed per head.  Keys visible to a position are
// numbered 0, 1, ...: the kept tokens before the window first, then the window, so that every kernel walks one range.
// Prompts in bf16 take slab_attention_sm100.cu; here are the norms of q and k, the form for any size and type, and the
// split-key form for a few new tokens.
#include <algorithm>

#include "decoder.cuh"
#include "warp_mma.cuh"

namespace {

// What position `pos` sees: `kept` leading tokens, then lo .. pos.
struct Visible {
  int lo, kept, n;
  __device__ __forceinline__ Visible(int pos, int window, int keep) {
    lo = max(0, pos - window + 1);
    kept = min(keep, lo);
    n = kept + pos - lo + 1;
  }
  __device__ __forceinline__ int key(int i) const { return i < kept ? i : lo + i - kept; }
};

// ---- norms of q and k, in place ---------------------------------------------------------------------------------------
// LG lanes per vector of `dim` entries: the heads * maps vectors of a row of q, then the kv_heads * maps of its new cache row.
template <typename T, int V, int LG>
__global__ void __launch_bounds__(256) k_qk_norm(T* __restrict__ q, long long ldq, T* __restrict__ kv, long long ld, int maxT, int first, int Tn,
                                                 int nq, int nk, int dim, const float* __restrict__ wq, const float* __restrict__ wk, float eps,
                                                 long long n) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & (LG - 1);
  long long it = (long long)blockIdx.x * (256 / LG) + threadIdx.x / LG;
  const bool live = it < n;
  if (!live) it = n - 1;
  const long long row = it / (nq + nk);
  const int i = (int)(it % (nq + nk));
  const float* w = i < nq ? wq : wk;
  T* x = i < nq ? q + row * ldq + (long long)i * dim
                : kv + ((row / Tn) * maxT + first + row % Tn) * ld + (long long)(i - nq) * dim;
  float ss = 0.f;
  for (int c = lane * V; c < dim; c += LG * V) {
    float f[V];
    load_vec<T, V>(x + c, f);
#pragma unroll
    for (int e = 0; e < V; e++) ss += f[e] * f[e];
  }
#pragma unroll
  for (int o = LG / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float inv = 1.f / sqrtf(ss / dim + eps);
  if (!live) return;
  for (int c = lane * V; c < dim; c += LG * V) {
    float f[V];
    load_vec<T, V>(x + c, f);
#pragma unroll
    for (int e = 0; e < V; e++) f[e] *= inv * w[c + e];
    store_vec<T, V>(x + c, f);
  }
}

// lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff
__global__ void k_diff_lambda(const float* lq1, const float* lk1, const float* lq2, const float* lk2, int dim, float diff, float* out) {
  float a = 0.f, b = 0.f;
  for (int i = threadIdx.x; i < dim; i += 32) { a = fmaf(lq1[i], lk1[i], a); b = fmaf(lq2[i], lk2[i], b); }
  a = warp_sum(a); b = warp_sum(b);
  if (threadIdx.x == 0) *out = expf(a) - expf(b) + diff;
}

// ---- a prompt, any size and type ----------------------------------------------------------------------------------------
// One block: 16 queries of one head; keys in tiles of 32 through shared memory, all arithmetic in fp32; the maps in turn.
constexpr int SQ = 16, SK = 32;
template <typename T, int MAPS>
__global__ void __launch_bounds__(128) k_window_attn(const WindowAttnArgs a) {
  extern __shared__ float sm[];
  const int D = a.dim, E = a.vdim, P = D + 1;
  float* qs = sm;                 // [SQ][P]
  float* ks = qs + SQ * P;        // [SK][P]
  float* vs = ks + SK * P;        // [SK][E]
  float* ps = vs + SK * E;        // [SQ][SK + 1]
  float* al = ps + SQ * (SK + 1); // [SQ]
  float* ls = al + SQ;            // [SQ]
  float* red = ls + SQ;           // [4]
  const int q0 = blockIdx.x * SQ, h = blockIdx.y, b = blockIdx.z, hk = h / (a.heads / a.kv_heads);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nq = min(SQ, a.T - q0);
  const T* kv = reinterpret_cast<const T*>(a.kv) + (long long)b * a.maxT * a.ld;
  const Visible oldest(a.first + q0, a.window, a.keep);
  const int n = oldest.n + nq - 1;      // numbered as the first query sees them, up to the last query's own key
  float acc[MAPS][2][SQ];
#pragma unroll
  for (int mp = 0; mp < MAPS; mp++) {
    float (&o0)[SQ] = acc[mp][0];
    float (&o1)[SQ] = acc[mp][1];
    __syncthreads();
    for (int i = tid; i < SQ * D; i += 128) {
      const int r = i / D, d = i % D;
      qs[r * P + d] = r < nq ? to_f<T>(reinterpret_cast<const T*>(a.q)[((long long)b * a.T + q0 + r) * a.ldq + (long long)(h * MAPS + mp) * D + d]) : 0.f;
    }
    float m[SQ / 4], l[SQ / 4];     // of the rows this warp owns
#pragma unroll
    for (int i = 0; i < SQ / 4; i++) { m[i] = -INFINITY; l[i] = 0.f; }
#pragma unroll
    for (int i = 0; i < SQ; i++) o0[i] = o1[i] = 0.f;
    for (int k0 = 0; k0 < n; k0 += SK) {
      const int nk = min(SK, n - k0);
      __syncthreads();
      for (int i = tid; i < nk * D; i += 128) {
        const int r = i / D, d = i % D;
        ks[r * P + d] = to_f<T>(kv[(long long)oldest.key(k0 + r) * a.ld + (long long)(hk * MAPS + mp) * D + d]);
      }
      for (int i = tid; i < nk * E; i += 128) {
        const int r = i / E, d = i % E;
        vs[r * E + d] = to_f<T>(kv[(long long)oldest.key(k0 + r) * a.ld + a.vo + (long long)hk * E + d]);
      }
      __syncthreads();
      const int j = oldest.key(k0 + lane);
#pragma unroll
      for (int i = 0; i < SQ / 4; i++) {
        const int r = warp * (SQ / 4) + i, pos = a.first + q0 + r;
        float s = -INFINITY;
        if (lane < nk && j <= pos && (pos - j < a.window || j < a.keep)) {
          s = 0.f;
          for (int d = 0; d < D; d++) s = fmaf(qs[r * P + d], ks[lane * P + d], s);
          s *= a.scale;
        }
        const float mn = fmaxf(m[i], warp_max(s));
        const float p = mn == -INFINITY ? 0.f : expf(s - mn), f = mn == -INFINITY ? 1.f : expf(m[i] - mn);
        l[i] = l[i] * f + warp_sum(p);
        m[i] = mn;
        ps[r * (SK + 1) + lane] = p;
        if (lane == 0) al[r] = f;
      }
      __syncthreads();
#pragma unroll
      for (int r = 0; r < SQ; r++) { o0[r] *= al[r]; o1[r] *= al[r]; }
      for (int k = 0; k < nk; k++) {
        const float v0 = tid < E ? vs[k * E + tid] : 0.f, v1 = tid + 128 < E ? vs[k * E + tid + 128] : 0.f;
#pragma unroll
        for (int r = 0; r < SQ; r++) {
          const float p = ps[r * (SK + 1) + k];
          o0[r] = fmaf(p, v0, o0[r]); o1[r] = fmaf(p, v1, o1[r]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < SQ / 4; i++) {
      float f = 1.f / l[i];
      if (a.sink) {
        const float z = a.sink[h], top = fmaxf(z, m[i]), e = expf(m[i] - top);
        f = e / (l[i] * e + expf(z - top));
      }
      if (lane == 0) ls[warp * (SQ / 4) + i] = f;
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < SQ; r++) { o0[r] *= ls[r]; o1[r] *= ls[r]; }
  }
  const T* gate = reinterpret_cast<const T*>(a.gate);
#pragma unroll
  for (int r = 0; r < SQ; r++) {
    float v0 = acc[0][0][r], v1 = acc[0][1][r];
    if (MAPS == 2) {
      const float lam = *a.lambda;
      v0 -= lam * acc[MAPS - 1][0][r]; v1 -= lam * acc[MAPS - 1][1][r];
      const float ss = warp_sum(v0 * v0 + v1 * v1);      // channels past vdim hold zeros
      __syncthreads();
      if (lane == 0) red[warp] = ss;
      __syncthreads();
      const float f = a.out_scale / sqrtf((red[0] + red[1] + red[2] + red[3]) / E + a.eps);
      v0 *= f; v1 *= f;
    }
    if (r >= nq) continue;
    const long long row = (long long)b * a.T + q0 + r;
    T* o = reinterpret_cast<T*>(a.o) + row * (long long)a.heads * E + (long long)h * E;
    const T* g = a.gate_mode == FEMTO_GATE_NONE ? nullptr : gate + row * a.ld_gate + (a.gate_mode == FEMTO_GATE_HEAD ? h : h * E);
    const bool each = a.gate_mode == FEMTO_GATE_ELEMENT;
    if (tid < E) o[tid] = from_f<T>(g ? v0 / (1.f + expf(-to_f<T>(g[each ? tid : 0]))) : v0);
    if (tid + 128 < E) o[tid + 128] = from_f<T>(g ? v1 / (1.f + expf(-to_f<T>(g[each ? tid + 128 : 0]))) : v1);
  }
}

// ---- a few new tokens ---------------------------------------------------------------------------------------------------
// grid (kv head x group of query heads, splits, rows).  A block takes `tiles_per` tiles of KT visible keys for up to VH
// (query head, map) pairs of its key/value head: the tile goes to shared memory, a warp does the scores of one pair against
// 32 keys, a warp the softmax of one pair, and the threads own channels of the result.  Partials (max, sum,
// unnormalised result) go to part[row][head][map][split][vdim + 2].
constexpr int VH = 16;
struct DecodeShape { int per, hq, groups, KT, pk, pv, splits, tiles_per; };   // pk, pv: elements between staged rows

template <typename T, bool VEC>
__device__ __forceinline__ void stage_rows(T* dst, int pitch, const T* src, long long ld, const Visible& vis, int i0, int n, int width, int tid) {
  if constexpr (VEC) {
    constexpr int V = VecN<T>::n;
    const int units = width / V;
    for (int i = tid; i < n * units; i += 256) {
      const int r = i / units, c = i % units * V;
      const uint32_t to = (uint32_t)__cvta_generic_to_shared(dst + r * pitch + c);
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to), "l"(src + (long long)vis.key(i0 + r) * ld + c) : "memory");
    }
  } else {
    for (int i = tid; i < n * width; i += 256) dst[i / width * pitch + i % width] = src[(long long)vis.key(i0 + i / width) * ld + i % width];
  }
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(256) k_window_decode(const WindowAttnArgs a, const DecodeShape sh) {
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t raw[];
  const int D = a.dim, E = a.vdim, KT = sh.KT;
  T* ks = reinterpret_cast<T*>(raw);                   // [KT][pk]
  T* vs = ks + KT * sh.pk;                             // [KT][pv]
  float* qs = reinterpret_cast<float*>(vs + KT * sh.pv);   // [VH][D]
  float* ss = qs + VH * ((D + 3) & ~3);                // [VH][KT]
  float* sal = ss + VH * KT;                           // [VH]
  float* sml = sal + VH;                               // [VH][2]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, LQ = (D + 3) & ~3;
  const int hk = blockIdx.x / sh.groups, h0 = hk * sh.per + blockIdx.x % sh.groups * sh.hq;
  const int nv = min(sh.hq, (hk + 1) * sh.per - h0) * a.maps;
  const long long row = blockIdx.z;
  const int b = (int)(row / a.T), pos = a.first + (int)(row % a.T);
  const Visible vis(pos, a.window, a.keep);
  const T* kv = reinterpret_cast<const T*>(a.kv) + (long long)b * a.maxT * a.ld;
  const T* ksrc = kv + (long long)hk * a.maps * D;
  const T* vsrc = kv + a.vo + (long long)hk * E;
  const T* q = reinterpret_cast<const T*>(a.q) + row * a.ldq + (long long)h0 * a.maps * D;
  pdl_wait();
  const int i0 = blockIdx.y * sh.tiles_per * KT, i1 = min(vis.n, i0 + sh.tiles_per * KT);
  for (int i = tid; i < nv * D; i += 256) qs[i / D * LQ + i % D] = to_f<T>(q[i]);
  if (tid < VH) { sml[2 * tid] = -INFINITY; sml[2 * tid + 1] = 0.f; }
  // results: thread -> channels c, c + 128; half of the pairs each, or, with few pairs, half of the keys each
  const int c = tid & 127, half = tid >> 7;
  const bool by_key = nv <= VH / 2;
  const int v0 = by_key ? 0 : half * (VH / 2), nvh = min(VH / 2, nv - v0);
  float acc[VH / 2][2];
#pragma unroll
  for (int i = 0; i < VH / 2; i++) acc[i][0] = acc[i][1] = 0.f;
  for (int t = i0; t < i1; t += KT) {
    const int n = min(KT, i1 - t);
    __syncthreads();
    stage_rows<T, VEC>(ks, sh.pk, ksrc, a.ld, vis, t, n, a.maps * D, tid);
    stage_rows<T, VEC>(vs, sh.pv, vsrc, a.ld, vis, t, n, E, tid);
    if (VEC) asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    const int blocks = KT / 32;
    for (int task = warp; task < nv * blocks; task += 8) {
      const int v = task / blocks, k = task % blocks * 32 + lane;
      float s = -INFINITY;
      if (k < n) {
        const T* kr = ks + k * sh.pk + v % a.maps * D;
        const float* qv = qs + v * LQ;
        float s0 = 0.f, s1 = 0.f;
        if constexpr (VEC) {
          constexpr int V = VecN<T>::n;
#pragma unroll 4
          for (int d = 0; d < D; d += V) {
            float f[V];
            load_vec<T, V>(kr + d, f);
#pragma unroll
            for (int e = 0; e < V; e += 4) {
              const float4 x = *reinterpret_cast<const float4*>(qv + d + e);
              s0 = fmaf(f[e], x.x, s0); s1 = fmaf(f[e + 1], x.y, s1); s0 = fmaf(f[e + 2], x.z, s0); s1 = fmaf(f[e + 3], x.w, s1);
            }
          }
        } else {
          for (int d = 0; d < D; d++) s0 = fmaf(to_f<T>(kr[d]), qv[d], s0);
        }
        s = (s0 + s1) * a.scale;
      }
      ss[v * KT + k] = s;
    }
    __syncthreads();
    for (int v = warp; v < nv; v += 8) {
      float m = sml[2 * v], mn = m;
      for (int k = lane; k < KT; k += 32) mn = fmaxf(mn, ss[v * KT + k]);
      mn = warp_max(mn);                               // finite: a tile holds at least one visible key
      float l = 0.f;
      for (int k = lane; k < KT; k += 32) {
        const float p = expf(ss[v * KT + k] - mn);
        ss[v * KT + k] = p;
        l += p;
      }
      l = warp_sum(l);
      __syncwarp();
      if (lane == 0) { const float f = expf(m - mn); sal[v] = f; sml[2 * v] = mn; sml[2 * v + 1] = sml[2 * v + 1] * f + l; }
    }
    __syncthreads();
    const int kb = by_key ? half * (KT / 2) : 0, ke = min(n, by_key ? kb + KT / 2 : KT);
#pragma unroll
    for (int i = 0; i < VH / 2; i++)
      if (i < nvh) { const float f = sal[v0 + i]; acc[i][0] *= f; acc[i][1] *= f; }
    if (c < E)
#pragma unroll 4
      for (int k = kb; k < ke; k++) {
        const float x = to_f<T>(vs[k * sh.pv + c]), y = c + 128 < E ? to_f<T>(vs[k * sh.pv + c + 128]) : 0.f;
#pragma unroll
        for (int i = 0; i < VH / 2; i++)
          if (i < nvh) { const float p = ss[(v0 + i) * KT + k]; acc[i][0] = fmaf(p, x, acc[i][0]); acc[i][1] = fmaf(p, y, acc[i][1]); }
      }
  }
  if (by_key) {      // the two halves of the keys, through the space of the keys' tile
    float* other = reinterpret_cast<float*>(raw);      // [VH / 2][E]
    __syncthreads();
    if (half) {
#pragma unroll
      for (int i = 0; i < VH / 2; i++)
        if (i < nvh) { if (c < E) other[i * E + c] = acc[i][0]; if (c + 128 < E) other[i * E + c + 128] = acc[i][1]; }
    }
    __syncthreads();
    if (!half) {
#pragma unroll
      for (int i = 0; i < VH / 2; i++)
        if (i < nvh) { if (c < E) acc[i][0] += other[i * E + c]; if (c + 128 < E) acc[i][1] += other[i * E + c + 128]; }
    }
  }
  __syncthreads();
  if (by_key && half) return;
#pragma unroll
  for (int i = 0; i < VH / 2; i++) {
    if (i >= nvh) break;
    const int v = v0 + i;
    float* dst = a.part + (((row * a.heads + h0) * a.maps + v) * sh.splits + blockIdx.y) * (E + 2);
    if (c == 0) { dst[0] = sml[2 * v]; dst[1] = sml[2 * v + 1]; }
    if (c < E) dst[2 + c] = acc[i][0];
    if (c + 128 < E) dst[2 + c + 128] = acc[i][1];
  }
}

// The tensor-core form for bf16: the pairs are the 16 rows of an mma tile, and each of the four warps of a block takes tiles of
// 32 visible keys of its own, which arrive in its part of shared memory by cp.async; the warps' results meet at the end.
// A query's row has zeros in the other map's channels, so that both maps run as one product with whole cached rows; the
// softmax weights are sums of two bf16 numbers and keep 32-bit accuracy.
// KS: steps of 16 key channels (maps dim <= 16 KS), NE: pairs of 8-channel tiles of the result (vdim <= 16 NE)
constexpr int DW = 4, DT = 32;      // warps of a block, keys of a tile
template <int KS, int NE>
__global__ void __launch_bounds__(32 * DW, KS <= 8 ? 3 : 1) k_window_decode_mma(const WindowAttnArgs a, const DecodeShape sh) {
  pdl_trigger();
  extern __shared__ __align__(16) uint8_t raw[];
  const int D = a.dim, E = a.vdim, MD = a.maps * D;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c2 = 2 * (lane & 3);
  bf16* ks = reinterpret_cast<bf16*>(raw) + warp * DT * (sh.pk + sh.pv);      // [DT][pk], swizzled
  bf16* vs = ks + DT * sh.pk;                                                // [DT][pv]
  const int hk = blockIdx.x / sh.groups, h0 = hk * sh.per + blockIdx.x % sh.groups * sh.hq;
  const int nv = min(sh.hq, (hk + 1) * sh.per - h0) * a.maps;
  const long long row = blockIdx.z;
  const int b = (int)(row / a.T), pos = a.first + (int)(row % a.T);
  const Visible vis(pos, a.window, a.keep);
  const bf16* kv = reinterpret_cast<const bf16*>(a.kv) + (long long)b * a.maxT * a.ld;
  const bf16* ksrc = kv + (long long)hk * MD;
  const bf16* vsrc = kv + a.vo + (long long)hk * E;
  const bf16* q = reinterpret_cast<const bf16*>(a.q) + row * a.ldq + (long long)h0 * MD;
  // the padding of the staged rows stays zero
  const uint4 zero = make_uint4(0, 0, 0, 0);
  for (int i = lane; i < DT * (sh.pk - MD) / 8; i += 32) { const int w = (sh.pk - MD) / 8; *reinterpret_cast<uint4*>(ks + swz(i / w, MD + i % w * 8, sh.pk)) = zero; }
  for (int i = lane; i < DT * (sh.pv - E) / 8; i += 32) { const int w = (sh.pv - E) / 8; *reinterpret_cast<uint4*>(vs + swz(i / w, E + i % w * 8, sh.pv)) = zero; }
  auto stage = [&](bf16* dst, int pitch, const bf16* src, int i0, int n, int units) {
    int r = lane / units, u = lane % units;
    const int dr = 32 / units, du = 32 % units;      // a step of 32 units
#pragma unroll 4
    while (r < DT) {
      if (r < n) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_addr(dst + swz(r, u * 8, pitch))), "l"(src + (long long)vis.key(i0 + r) * a.ld + u * 8) : "memory");
      else *reinterpret_cast<uint4*>(dst + swz(r, u * 8, pitch)) = zero;
      r += dr; u += du;
      if (u >= units) { u -= units; r++; }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  const int first = blockIdx.y * sh.tiles_per, last = min(first + sh.tiles_per, (vis.n + DT - 1) / DT);
  pdl_wait();
  uint32_t qa[KS][4];
  float o[NE][2][4] = {}, m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  for (int t = first + warp; t < last; t += DW) {
    const int n = min(DT, vis.n - t * DT);
    __syncwarp();
    stage(ks, sh.pk, ksrc, t * DT, n, MD / 8);
    stage(vs, sh.pv, vsrc, t * DT, n, E / 8);
    if (t == first + warp) {
#pragma unroll
      for (int k = 0; k < KS; k++)
#pragma unroll
        for (int e = 0; e < 4; e++) {
          const int v = g + 8 * (e & 1), c = k * 16 + 8 * (e >> 1) + c2 - (a.maps == 2 ? v % 2 * D : 0);
          qa[k][e] = v < nv && c >= 0 && c < D ? *reinterpret_cast<const uint32_t*>(q + v * D + c) : 0u;
        }
    }
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncwarp();
    float s[4][4] = {};
#pragma unroll
    for (int k = 0; k < KS; k++) {
      if (k * 16 >= MD) break;
#pragma unroll
      for (int j = 0; j < 2; j++) {
        uint32_t kb[4];
        ldsm4(kb, ks + swz(16 * j + (lane & 7) + 8 * (lane >> 4), k * 16 + 8 * ((lane >> 3) & 1), sh.pk));
        mma16816(s[2 * j], qa[k], kb[0], kb[1]);
        mma16816(s[2 * j + 1], qa[k], kb[2], kb[3]);
      }
    }
    // softmax of rows g and g + 8, each shared by four lanes
    float f[2];
#pragma unroll
    for (int e = 0; e < 2; e++) {
      float mn = m[e];
#pragma unroll
      for (int j = 0; j < 4; j++)
#pragma unroll
        for (int i = 0; i < 2; i++) {
          float& x = s[j][2 * e + i];
          x = 8 * j + c2 + i < n ? x * a.scale : -INFINITY;
          mn = fmaxf(mn, x);
        }
      mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, 1));
      mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, 2));      // finite: a tile holds at least one visible key
      f[e] = __expf(m[e] - mn);
      m[e] = mn;
      l[e] *= f[e];
#pragma unroll
      for (int j = 0; j < 4; j++)
#pragma unroll
        for (int i = 0; i < 2; i++) { float& x = s[j][2 * e + i]; x = __expf(x - mn); l[e] += x; }
    }
#pragma unroll
    for (int j = 0; j < NE; j++)
#pragma unroll
      for (int i = 0; i < 2; i++) { o[j][i][0] *= f[0]; o[j][i][1] *= f[0]; o[j][i][2] *= f[1]; o[j][i][3] *= f[1]; }
    uint32_t ph[2][4], pl[2][4];
#pragma unroll
    for (int k = 0; k < 2; k++)
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const float x = s[2 * k + (e >> 1)][2 * (e & 1)], y = s[2 * k + (e >> 1)][2 * (e & 1) + 1];
        const __nv_bfloat162 hi = __floats2bfloat162_rn(x, y);
        const __nv_bfloat162 lo = __floats2bfloat162_rn(x - __bfloat162float(hi.x), y - __bfloat162float(hi.y));
        ph[k][e] = *reinterpret_cast<const uint32_t*>(&hi);
        pl[k][e] = *reinterpret_cast<const uint32_t*>(&lo);
      }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncwarp();
#pragma unroll
    for (int j = 0; j < NE; j++) {
      if (j * 16 >= E) break;
#pragma unroll
      for (int k = 0; k < 2; k++) {
        uint32_t vb[4];
        ldsm4t(vb, vs + swz(16 * k + (lane & 15), j * 16 + 8 * (lane >> 4), sh.pv));
#pragma unroll
        for (int i = 0; i < 2; i++) { mma16816(o[j][i], ph[k], vb[2 * i], vb[2 * i + 1]); mma16816(o[j][i], pl[k], vb[2 * i], vb[2 * i + 1]); }
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 2; e++) {
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
  }
  // the warps' results through shared memory: [DW][16][E], and their maxima and sums
  __shared__ float sm[DW][16], sl[DW][16];
  float* os = reinterpret_cast<float*>(raw);
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 2; e++) {
    const int v = g + 8 * e;
    if ((lane & 3) == 0) { sm[warp][v] = m[e]; sl[warp][v] = l[e]; }
#pragma unroll
    for (int j = 0; j < NE; j++)
#pragma unroll
      for (int i = 0; i < 2; i++) {
        const int c = j * 16 + 8 * i + c2;
        if (v < nv && c < E) *reinterpret_cast<float2*>(os + (warp * 16 + v) * E + c) = make_float2(o[j][i][2 * e], o[j][i][2 * e + 1]);
      }
  }
  __syncthreads();
  for (int i = tid; i < nv * E; i += 32 * DW) {
    const int v = i / E, c = i % E;
    float M = -INFINITY, L = 0.f, x = 0.f;
#pragma unroll
    for (int w = 0; w < DW; w++) M = fmaxf(M, sm[w][v]);
#pragma unroll
    for (int w = 0; w < DW; w++) {
      const float r = sm[w][v] == -INFINITY ? 0.f : __expf(sm[w][v] - M);
      L += r * sl[w][v];
      x = fmaf(r, os[(w * 16 + v) * E + c], x);
    }
    float* dst = a.part + (((row * a.heads + h0) * a.maps + v) * sh.splits + blockIdx.y) * (E + 2);
    if (c == 0) { dst[0] = M; dst[1] = L; }
    dst[2 + c] = x;
  }
}

// grid (heads, rows): the splits of a head, the sink, the difference of the maps and its norm, the gate.  Four groups of 128
// threads take every fourth split.
template <typename T, int MAPS>
__global__ void __launch_bounds__(512) k_window_combine(const WindowAttnArgs a, int splits) {
  pdl_trigger();
  extern __shared__ float sm[];
  float* ws = sm;                 // [MAPS][splits]
  __shared__ float os[3][MAPS][256], red[4];
  const int h = blockIdx.x, tid = threadIdx.x & 127, part = threadIdx.x >> 7, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, E = a.vdim;
  const long long row = blockIdx.y;
  const T* gp = reinterpret_cast<const T*>(a.gate) + (a.gate_mode == FEMTO_GATE_NONE ? 0 : row * a.ld_gate + (a.gate_mode == FEMTO_GATE_HEAD ? h : h * E));
  const float* p = a.part + (row * a.heads + h) * MAPS * (long long)splits * (E + 2);
  const float z = a.sink ? a.sink[h] : -INFINITY, lam = MAPS == 2 ? *a.lambda : 0.f;
  pdl_wait();
  float gate[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 2; i++)
    if (!part && tid + 128 * i < E && a.gate_mode != FEMTO_GATE_NONE) gate[i] = to_f<T>(gp[a.gate_mode == FEMTO_GATE_HEAD ? 0 : tid + 128 * i]);
  if (warp < MAPS) {
    const float* pm = p + (long long)warp * splits * (E + 2);
    float M = z, L = 0.f;
    for (int s = lane; s < splits; s += 32) { const float m = pm[(long long)s * (E + 2)]; ws[warp * splits + s] = m; M = fmaxf(M, m); }
    M = warp_max(M);
    for (int s = lane; s < splits; s += 32) {
      const float w = expf(ws[warp * splits + s] - M);      // an empty split: exp(-inf) = 0
      L += w * pm[(long long)s * (E + 2) + 1];
      ws[warp * splits + s] = w;
    }
    L = warp_sum(L);
    if (a.sink) L += expf(z - M);
    L = 1.f / L;
    __syncwarp();
    for (int s = lane; s < splits; s += 32) ws[warp * splits + s] *= L;
  }
  __syncthreads();
  float o[MAPS][2];
#pragma unroll
  for (int mp = 0; mp < MAPS; mp++) {
    const float* pm = p + (long long)mp * splits * (E + 2) + 2;
#pragma unroll
    for (int i = 0; i < 2; i++) {
      o[mp][i] = 0.f;
      const int c = tid + 128 * i;
      if (c < E)
#pragma unroll 4
        for (int s = part; s < splits; s += 4) o[mp][i] = fmaf(ws[mp * splits + s], pm[(long long)s * (E + 2) + c], o[mp][i]);
      if (part) os[part - 1][mp][c] = o[mp][i];
    }
  }
  __syncthreads();
  if (part) return;
  float v[2];
#pragma unroll
  for (int i = 0; i < 2; i++) {
#pragma unroll
    for (int mp = 0; mp < MAPS; mp++) o[mp][i] += (os[0][mp][tid + 128 * i] + os[1][mp][tid + 128 * i]) + os[2][mp][tid + 128 * i];
    v[i] = MAPS == 2 ? o[0][i] - lam * o[MAPS - 1][i] : o[0][i];
  }
  if (MAPS == 2) {
    const float ss = warp_sum(v[0] * v[0] + v[1] * v[1]);      // channels past vdim hold zeros
    if (lane == 0) red[warp] = ss;
    asm volatile("bar.sync 1, 128;" ::: "memory");
    const float f = a.out_scale / sqrtf((red[0] + red[1] + red[2] + red[3]) / E + a.eps);
    v[0] *= f; v[1] *= f;
  }
  T* o_row = reinterpret_cast<T*>(a.o) + row * (long long)a.heads * E + (long long)h * E;
#pragma unroll
  for (int i = 0; i < 2; i++) {
    const int c = tid + 128 * i;
    if (c >= E) continue;
    if (a.gate_mode != FEMTO_GATE_NONE) v[i] /= 1.f + expf(-gate[i]);
    o_row[c] = from_f<T>(v[i]);
  }
}

template <typename K> int allow_smem(K kernel, size_t bytes) {
  if (bytes > 227 * 1024) return femto_fail(FEMTO_ERR_UNSUPPORTED, "attention: a tile needs %zu bytes of shared memory", bytes);
  if (bytes > 48 * 1024) CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
  return 0;
}

template <typename T> int window_decode(const WindowAttnArgs& a, cudaStream_t s) {
  constexpr int V = VecN<T>::n;
  const int rows = a.B * a.T, es = sizeof(T);
  DecodeShape sh;
  sh.per = a.heads / a.kv_heads;
  sh.hq = std::min(sh.per, VH / a.maps);
  sh.groups = cdiv(sh.per, sh.hq);
  const bool vec = a.dim % V == 0 && a.vdim % V == 0 && a.ld % V == 0 && a.vo % V == 0 && aligned16(a.kv);
  const bool tc = es == 2 && vec && a.maps * a.dim <= 256 && a.vdim <= 256 && (a.ldq & 1) == 0;
  const int seen = (int)std::min<long long>(a.first + a.T, (long long)a.window + a.keep), blocks = a.kv_heads * sh.groups * rows;
  size_t smem;
  int tiles;
  if (tc) {
    sh.pk = round_up(a.maps * a.dim, 64); sh.pv = round_up(a.vdim, 64); sh.KT = DT;
    smem = (size_t)2 * DW * DT * (sh.pk + sh.pv);
    tiles = cdiv(seen, DT);
    // a block's four warps have a tile each, more when that makes more blocks than run at once
    sh.tiles_per = std::max(DW, cdiv(tiles, std::max(1, 3 * device_sm_count() / blocks)));
  } else {
    // odd numbers of 16-byte units between staged rows keep the vector loads of neighbouring keys on different banks
    sh.pk = (cdiv(a.maps * a.dim * es, 16) | 1) * V;
    sh.pv = (cdiv(a.vdim * es, 16) | 1) * V;
    auto bytes = [&](int kt) {
      return std::max((size_t)es * kt * (sh.pk + sh.pv) + 4 * (size_t)(VH * ((a.dim + 3) & ~3) + VH * kt + 3 * VH), (size_t)4 * (VH / 2) * a.vdim);
    };
    sh.KT = bytes(64) <= 200 * 1024 ? 64 : 32;
    smem = bytes(sh.KT);
    tiles = cdiv(seen, sh.KT);
    sh.tiles_per = cdiv(tiles, std::max(1, std::min(tiles, cdiv(2 * device_sm_count(), blocks))));
  }
  auto floats = [&] { return (size_t)rows * a.heads * a.maps * cdiv(tiles, sh.tiles_per) * (a.vdim + 2); };
  while (floats() > a.part_floats && sh.tiles_per < tiles) sh.tiles_per++;
  if (floats() > a.part_floats) return femto_fail(FEMTO_ERR_STATE, "attention: no room for the partial results of %d rows", rows);
  sh.splits = cdiv(tiles, sh.tiles_per);
  const dim3 grid(a.kv_heads * sh.groups, sh.splits, rows);
#define LAUNCH(KERNEL, THREADS) do { FEMTO_TRY(allow_smem(KERNEL, smem)); CUDA_TRY(launch_dependent(KERNEL, grid, THREADS, smem, s, a, sh)); } while (0)
  if (tc) {
    if (sh.pk <= 64 && sh.pv <= 64) LAUNCH((k_window_decode_mma<4, 4>), 32 * DW);
    else if (sh.pk <= 128 && sh.pv <= 128) LAUNCH((k_window_decode_mma<8, 8>), 32 * DW);
    else LAUNCH((k_window_decode_mma<16, 16>), 32 * DW);
  } else if (vec) LAUNCH((k_window_decode<T, true>), 256);
  else LAUNCH((k_window_decode<T, false>), 256);
#undef LAUNCH
  KERNEL_CHECK();
  const size_t ws = 4 * (size_t)a.maps * sh.splits;
  if (a.maps == 2) CUDA_TRY(launch_dependent(k_window_combine<T, 2>, dim3(a.heads, rows), 512, ws, s, a, sh.splits));
  else CUDA_TRY(launch_dependent(k_window_combine<T, 1>, dim3(a.heads, rows), 512, ws, s, a, sh.splits));
  KERNEL_CHECK();
  return 0;
}

}  // namespace

size_t window_attention_part_floats(int max_batch, int heads, int maps, int vdim) {
  return (size_t)heads * maps * (vdim + 2) * ((size_t)max_batch * ATTN_FEW + 3 * 160);
}

int diff_lambda(const float* lq1, const float* lk1, const float* lq2, const float* lk2, int dim, float diff, float* out, cudaStream_t s) {
  k_diff_lambda<<<1, 32, 0, s>>>(lq1, lk1, lq2, lk2, dim, diff, out);
  KERNEL_CHECK();
  return 0;
}

template <typename T> int qk_norm(const WindowAttnArgs& a, const float* wq, const float* wk, bool with_k, cudaStream_t s) {
  constexpr int V = VecN<T>::n;
  const int nq = a.heads * a.maps, nk = with_k ? a.kv_heads * a.maps : 0;
  const long long n = (long long)a.B * a.T * (nq + nk);
  T *q = (T*)const_cast<void*>(a.q), *kv = (T*)const_cast<void*>(a.kv);
  const bool vec = a.dim % V == 0 && a.ldq % V == 0 && a.ld % V == 0 && aligned16(a.q) && aligned16(a.kv);
#define LAUNCH(VV, LG) CUDA_TRY(launch_dependent(k_qk_norm<T, VV, LG>, cdiv(n, 256 / LG), 256, 0, s, q, a.ldq, kv, (long long)a.ld, a.maxT, a.first, a.T, nq, nk, \
                                                 a.dim, wq, wk, a.eps, n))
  if (!vec) LAUNCH(1, 32);
  else if (a.dim <= 8 * V) LAUNCH(V, 8);
  else if (a.dim <= 16 * V) LAUNCH(V, 16);
  else LAUNCH(V, 32);
#undef LAUNCH
  KERNEL_CHECK();
  return 0;
}
template int qk_norm<float>(const WindowAttnArgs&, const float*, const float*, bool, cudaStream_t);
template int qk_norm<bf16>(const WindowAttnArgs&, const float*, const float*, bool, cudaStream_t);

template <typename T> int window_attention(const WindowAttnArgs& a, cudaStream_t s) {
  if (a.T <= ATTN_FEW) return window_decode<T>(a, s);
  if (sizeof(T) == 2 && window_attention_tc_supported(a)) return window_attention_tc(a, s);
  const size_t smem = 4 * (size_t)((SQ + SK) * (a.dim + 1) + SK * a.vdim + SQ * (SK + 1) + 2 * SQ + 4);
  const dim3 grid(cdiv(a.T, SQ), a.heads, a.B);
  if (a.maps == 2) {
    FEMTO_TRY(allow_smem(k_window_attn<T, 2>, smem));
    k_window_attn<T, 2><<<grid, 128, smem, s>>>(a);
  } else {
    FEMTO_TRY(allow_smem(k_window_attn<T, 1>, smem));
    k_window_attn<T, 1><<<grid, 128, smem, s>>>(a);
  }
  KERNEL_CHECK();
  return 0;
}
template int window_attention<float>(const WindowAttnArgs&, cudaStream_t);
template int window_attention<bf16>(const WindowAttnArgs&, cudaStream_t);

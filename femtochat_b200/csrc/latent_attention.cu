// Attention over a cached low-rank latent: every token leaves one row [latent | rotated key part] that all heads share.
// A prompt expands the latents of its keys into per-head keys and values once and attends as usual; a few new tokens
// attend in the latent space instead, with queries taken through the key up-projection and the result through the value
// up-projection, so that a decode step reads each cached row once for all heads.
#include <algorithm>

#include "decoder.cuh"
#include "warp_mma.cuh"

namespace {

// ---- new rows ---------------------------------------------------------------------------------------------------------
// out[0 .. ldo) = rms_norm(in[0 .. size)) w, then zeros; by one warp
template <typename T, int V>
__device__ __forceinline__ void warp_norm(const T* __restrict__ in, const float* __restrict__ w, T* __restrict__ out, int ldo, int size,
                                          float eps, int lane) {
  float ss = 0.f;
#pragma unroll 4
  for (int c = lane * V; c < size; c += 32 * V) {
    float f[V];
    load_vec<T, V>(in + c, f);
#pragma unroll
    for (int e = 0; e < V; e++) ss += f[e] * f[e];
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / size + eps);
#pragma unroll 4
  for (int c = lane * V; c < ldo; c += 32 * V) {
    float f[V] = {};
    if (c < size) load_vec<T, V>(in + c, f);
#pragma unroll
    for (int e = 0; e < V; e++) f[e] = c + e < size ? f[e] * inv * w[c + e] : 0.f;
    store_vec<T, V>(out + c, f);
  }
}
__device__ __forceinline__ void rotate(float u, float v, float pos, float freq, float& a, float& b) {
  float sn, cs;
  sincosf(pos * freq, &sn, &cs);
  a = u * cs - v * sn;
  b = v * cs + u * sn;
}

// One warp per (row, part): part 0 norms the query latent, part 1 norms the latent and rotates the shared key part into
// the cache.
template <typename T>
__global__ void __launch_bounds__(256) k_latent_norms(const LatentArgs a) {
  pdl_trigger();
  pdl_wait();
  constexpr int V = VecN<T>::n;
  const long long it = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (it >= 2LL * a.B * a.T) return;
  const int lane = threadIdx.x & 31, part = (int)(it & 1);
  const long long row = it >> 1;
  if (part == 0) {
    const T* src = reinterpret_cast<const T*>(a.dq) + row * a.ld_dkv;
    T* dst = reinterpret_cast<T*>(a.cq) + row * a.qp;
    if (a.q_rank % V == 0) warp_norm<T, V>(src, a.dq_norm, dst, a.qp, a.q_rank, a.eps, lane);
    else warp_norm<T, 1>(src, a.dq_norm, dst, a.qp, a.q_rank, a.eps, lane);
    return;
  }
  const int b = (int)(row / a.T), t = (int)(row % a.T);
  const T* src = reinterpret_cast<const T*>(a.dkv) + row * a.ld_dkv;
  T* dst = reinterpret_cast<T*>(a.latent) + ((long long)b * a.maxT + a.first + t) * a.ld;
  if (a.kv_rank % V == 0) warp_norm<T, V>(src, a.dkv_norm, dst, a.lp, a.kv_rank, a.eps, lane);
  else warp_norm<T, 1>(src, a.dkv_norm, dst, a.lp, a.kv_rank, a.eps, lane);
  const int half = a.rot_dims / 2;
  src += a.kv_rank;
  dst += a.lp;
  for (int i = lane; i < half; i += 32) {
    float u, v;
    rotate(to_f<T>(src[i]), to_f<T>(src[i + half]), (float)(a.first + t), a.freq[i], u, v);
    dst[i] = from_f<T>(u);
    dst[i + half] = from_f<T>(v);
  }
  for (int i = a.rot_dims + lane; i < a.rot_dim; i += 32) dst[i] = src[i];
}

// q in place, for prompts: a thread rotates V neighbouring pairs of every head of its row (V = 2 needs even offsets).
template <typename T, int V>
__global__ void __launch_bounds__(256) k_rotate_q(const LatentArgs a) {
  pdl_trigger();
  pdl_wait();
  struct __align__(V * sizeof(T)) Vec { T v[V]; };
  const int half = a.rot_dims / 2, hd = a.dim + a.rot_dim, per = half / V;
  const long long it = (long long)blockIdx.x * 256 + threadIdx.x;
  if (it >= (long long)a.B * a.T * per) return;
  const int i = (int)(it % per) * V;
  const long long row = it / per;
  float sn[V], cs[V];
#pragma unroll
  for (int e = 0; e < V; e++) sincosf((float)(a.first + (int)(row % a.T)) * a.freq[i + e], &sn[e], &cs[e]);
  T* q = reinterpret_cast<T*>(a.q) + row * (long long)a.heads * hd + a.dim;
#pragma unroll 8
  for (int h = 0; h < a.heads; h++, q += hd) {
    Vec u = *reinterpret_cast<const Vec*>(q + i), v = *reinterpret_cast<const Vec*>(q + i + half);
#pragma unroll
    for (int e = 0; e < V; e++) {
      const float x = to_f<T>(u.v[e]), y = to_f<T>(v.v[e]);
      u.v[e] = from_f<T>(x * cs[e] - y * sn[e]);
      v.v[e] = from_f<T>(y * cs[e] + x * sn[e]);
    }
    *reinterpret_cast<Vec*>(q + i) = u;
    *reinterpret_cast<Vec*>(q + i + half) = v;
  }
}

// ---- a prompt: expanded keys and values -----------------------------------------------------------------------------
// One block: 16 queries of one head; keys in tiles of 32 through shared memory, all arithmetic in fp32.
constexpr int SQ = 16, SK = 32;
template <typename T>
__global__ void __launch_bounds__(128) k_latent_attn_simt(const LatentArgs a, int N) {
  extern __shared__ float sm[];
  const int Dk = a.dim + a.rot_dim, E = a.vdim, P = Dk + 1;
  float* qs = sm;                 // [SQ][P]
  float* ks = qs + SQ * P;        // [SK][P]
  float* vs = ks + SK * P;        // [SK][E]
  float* ps = vs + SK * E;        // [SQ][SK + 1]
  float* al = ps + SQ * (SK + 1); // [SQ]
  float* ls = al + SQ;            // [SQ]
  const int q0 = blockIdx.x * SQ, h = blockIdx.y, b = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nq = min(SQ, a.T - q0);
  const long long ldkv = (long long)a.heads * (a.dim + a.vdim);
  const T* kv = reinterpret_cast<const T*>(a.kv) + (long long)b * a.maxT * ldkv;
  const T* lat = reinterpret_cast<const T*>(a.latent) + (long long)b * a.maxT * a.ld + a.lp;
  for (int i = tid; i < SQ * Dk; i += 128) {
    const int r = i / Dk, d = i % Dk;
    qs[r * P + d] = r < nq ? to_f<T>(reinterpret_cast<const T*>(a.q)[(((long long)b * a.T + q0 + r) * a.heads + h) * Dk + d]) : 0.f;
  }
  float m[SQ / 4], l[SQ / 4];     // of the rows this warp owns
#pragma unroll
  for (int i = 0; i < SQ / 4; i++) { m[i] = -INFINITY; l[i] = 0.f; }
  float o0[SQ], o1[SQ];
#pragma unroll
  for (int i = 0; i < SQ; i++) o0[i] = o1[i] = 0.f;
  const int last = a.first + q0 + nq - 1;
  for (int k0 = 0; k0 <= last; k0 += SK) {
    const int nk = min(SK, N - k0);
    __syncthreads();
    for (int i = tid; i < nk * Dk; i += 128) {
      const int r = i / Dk, d = i % Dk;
      ks[r * P + d] = to_f<T>(d < a.dim ? kv[(k0 + r) * ldkv + (long long)h * a.dim + d] : lat[(long long)(k0 + r) * a.ld + d - a.dim]);
    }
    for (int i = tid; i < nk * E; i += 128) {
      const int r = i / E, d = i % E;
      vs[r * E + d] = to_f<T>(kv[(k0 + r) * ldkv + (long long)a.heads * a.dim + (long long)h * E + d]);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < SQ / 4; i++) {
      const int r = warp * (SQ / 4) + i;
      float s = -INFINITY;
      if (lane < nk && k0 + lane <= a.first + q0 + r) {
        s = 0.f;
        for (int d = 0; d < Dk; d++) s = fmaf(qs[r * P + d], ks[lane * P + d], s);
        s *= a.scale;
      }
      const float mn = fmaxf(m[i], warp_max(s));
      const float p = mn == -INFINITY ? 0.f : expf(s - mn), f = mn == -INFINITY ? 1.f : expf(m[i] - mn);
      l[i] = l[i] * f + warp_sum(p);
      m[i] = mn;
      ps[r * (SK + 1) + lane] = p;
      if (lane == 0) { al[r] = f; ls[r] = l[i]; }
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
  for (int r = 0; r < SQ; r++) {
    if (r >= nq) break;
    const long long row = (long long)b * a.T + q0 + r;
    const float g = to_f<T>(reinterpret_cast<const T*>(a.gate)[row * a.ld_gate + h]);
    const float f = 1.f / (ls[r] * (1.f + expf(-g)));
    T* o = reinterpret_cast<T*>(a.o) + row * (long long)a.heads * E + (long long)h * E;
    if (tid < E) o[tid] = from_f<T>(o0[r] * f);
    if (tid + 128 < E) o[tid + 128] = from_f<T>(o1[r] * f);
  }
}

// ---- a few tokens: attention in the latent space ----------------------------------------------------------------------
// qabs[row][head] = [W_uk^T q (kv_rank), zeros up to lp, rotated q (rot_dim), zeros up to ld].  A thread owns one 16-byte
// group of latent channels and one slice of the head's channels.
template <typename T>
__global__ void __launch_bounds__(1024) k_absorb_q(const LatentArgs a) {
  pdl_trigger();
  pdl_wait();
  constexpr int V = VecN<T>::n;
  extern __shared__ float sm[];
  const int h = blockIdx.x, hd = a.dim + a.rot_dim, tid = threadIdx.x;
  const long long row = blockIdx.y;
  float* qs = sm;                     // [hd]
  float* part = sm + hd;              // [slices][lp]
  const T* q = reinterpret_cast<const T*>(a.q) + (row * a.heads + h) * hd;
  for (int i = tid; i < hd; i += 1024) qs[i] = to_f<T>(q[i]);
  __syncthreads();
  const int groups = a.lp / V, slices = 1024 / groups, per = (a.dim + slices - 1) / slices;
  const int gr = tid % groups, sl = tid / groups;
  if (sl < slices) {
    float acc[V] = {};
    const int d1 = min(a.dim, (sl + 1) * per);
    const T* w = reinterpret_cast<const T*>(a.w_kv) + (long long)h * a.dim * a.lp + gr * V;
#pragma unroll 8
    for (int d = sl * per; d < d1; d++) {
      float f[V];
      load_vec<T, V>(w + (long long)d * a.lp, f);
#pragma unroll
      for (int e = 0; e < V; e++) acc[e] = fmaf(qs[d], f[e], acc[e]);
    }
#pragma unroll
    for (int e = 0; e < V; e++) part[sl * a.lp + gr * V + e] = acc[e];
  }
  __syncthreads();
  float* dst = a.qabs + (row * a.heads + h) * a.ld;
  const int half = a.rot_dims / 2;
  for (int c = tid; c < a.ld; c += 1024) {
    float x = 0.f;
    if (c < a.lp) {
      for (int k = 0; k < slices; k++) x += part[k * a.lp + c];
    } else if (c < a.lp + a.rot_dim) {
      const int i = c - a.lp;
      const float* qr = qs + a.dim;
      x = qr[i];
      if (i < a.rot_dims) {
        float u, v;
        const int k = i < half ? i : i - half;
        rotate(qr[k], qr[k + half], (float)(a.first + (int)(row % a.T)), a.freq[k], u, v);
        x = round_to<T>(i < half ? u : v);
      }
    }
    dst[c] = x;
  }
}

// The tensor-core form for bf16 caches.  grid (heads / 16, splits, rows): 16 heads are the rows of one mma tile; the cached
// rows arrive in tiles of `KT` through two shared-memory buffers (16-byte units of row r permuted by r & 7) and serve as
// keys (read as they lie) and as values (read transposed).  Queries and softmax weights are sums of two bf16 numbers, so
// scores and weights keep fp32 accuracy.  For the scores the warps share the channels, so a warp's part of the queries
// stays in registers for the whole kernel and shared memory is read once; their partial sums meet in shared memory.
// NK: 16-channel steps per warp (width <= 128 NK); NP: pairs of 8-channel tiles of the result per warp (lp <= 128 NP)
template <int NK, int NP>
__global__ void __launch_bounds__(256) k_latent_decode_mma(const LatentArgs a, int splits, int tiles_per, int KT, int width) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t raw[];
  const int SP = KT + 4;
  bf16* rows = reinterpret_cast<bf16*>(raw);            // 2 x [KT][width]
  bf16* ph = rows + 2 * KT * width;                     // [16][64] high, low
  float* ss = reinterpret_cast<float*>(ph + 2 * 16 * 64);   // [8 warps][16][SP]
  float* sal = ss + 8 * 16 * SP;                        // [16] rescale factor of this tile
  float* sml = sal + 16;                                // [16][2] running max and sum
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, c2 = 2 * (lane & 3);
  const int h0 = blockIdx.x * 16, sp = blockIdx.y;
  const long long row = blockIdx.z;
  const int b = (int)(row / a.T), n = a.first + (int)(row % a.T) + 1;      // keys this query sees
  const int ntiles = (n + KT - 1) / KT, tb = sp * tiles_per, te = min(ntiles, tb + tiles_per);
  const bf16* lat = reinterpret_cast<const bf16*>(a.latent) + (long long)b * a.maxT * a.ld;
  const int units = a.ld / 8;
  auto load = [&](int tile) {
    bf16* dst = rows + (tile & 1) * KT * width;
    for (int i = tid; i < KT * units; i += 256) {
      const int r = i / units, c = i % units * 8, key = tile * KT + r;
      const uint32_t to = smem_addr(dst + swz(r, c, width));
      if (key < n) asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to), "l"(lat + (long long)key * a.ld + c) : "memory");
      else *reinterpret_cast<uint4*>(dst + swz(r, c, width)) = make_uint4(0, 0, 0, 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (tb < te) load(tb);
  // the rotated parts of the queries, through shared memory that the scores use later
  float* qr = ss;                                       // [16][rot_dim]
  const int half = a.rot_dims / 2, rest = a.rot_dim - half;       // a thread makes both entries of a pair, or passes one on
  for (int i = tid; i < 16 * rest; i += 256) {
    const int r = i / rest, k = i % rest, h = h0 + r;
    if (h >= a.heads) continue;
    const bf16* q = reinterpret_cast<const bf16*>(a.q) + (row * a.heads + h) * (a.dim + a.rot_dim) + a.dim;
    if (k < half) {
      float u, v;
      rotate(__bfloat162float(q[k]), __bfloat162float(q[k + half]), (float)(n - 1), a.freq[k], u, v);
      qr[r * a.rot_dim + k] = round_to<bf16>(u);
      qr[r * a.rot_dim + k + half] = round_to<bf16>(v);
    } else {
      qr[r * a.rot_dim + k + half] = __bfloat162float(q[k + half]);
    }
  }
  __syncthreads();
  // this warp's steps of the queries: latent channels from qabs, then the rotated part, zeros in the padding
  uint32_t qa[NK][4], ql[NK][4];
#pragma unroll
  for (int s = 0; s < NK; s++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int r = g + 8 * (e & 1), h = h0 + r, c = (warp + 8 * s) * 16 + 8 * (e >> 1) + c2;
      float2 f = make_float2(0.f, 0.f);
      if (h < a.heads) {
        if (c < a.lp) {
          f = *reinterpret_cast<const float2*>(a.qabs + (row * a.heads + h) * a.lp + c);
        } else {
          if (c < a.lp + a.rot_dim) f.x = qr[r * a.rot_dim + c - a.lp];
          if (c + 1 < a.lp + a.rot_dim) f.y = qr[r * a.rot_dim + c + 1 - a.lp];
        }
      }
      const __nv_bfloat162 hi = __floats2bfloat162_rn(f.x, f.y);
      const __nv_bfloat162 lo = __floats2bfloat162_rn(f.x - __bfloat162float(hi.x), f.y - __bfloat162float(hi.y));
      qa[s][e] = *reinterpret_cast<const uint32_t*>(&hi);
      ql[s][e] = *reinterpret_cast<const uint32_t*>(&lo);
    }
  const int pad = width - a.ld;
  if (pad)
    for (int i = tid; i < 2 * KT * pad / 8; i += 256) {
      const int r = i / (pad / 8), c = a.ld + i % (pad / 8) * 8;
      *reinterpret_cast<uint4*>(rows + (r / KT) * KT * width + swz(r % KT, c, width)) = make_uint4(0, 0, 0, 0);
    }
  if (tid < 16) { sml[2 * tid] = -INFINITY; sml[2 * tid + 1] = 0.f; }
  float o[NP][2][4] = {};
  for (int tile = tb; tile < te; tile++) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                   // the tile is complete, the other buffer free
    if (tile + 1 < te) load(tile + 1);
    const bf16* kt = rows + (tile & 1) * KT * width;
    for (int j = 0; j < KT; j += 16) { // partial scores of 16 keys
      float s[2][4] = {};
#pragma unroll
      for (int k = 0; k < NK; k++) {
        const int c = (warp + 8 * k) * 16;
        if (c >= width) break;
        uint32_t kb[4];
        ldsm4(kb, kt + swz(j + (lane & 7) + 8 * (lane >> 4), c + 8 * ((lane >> 3) & 1), width));
#pragma unroll
        for (int i = 0; i < 2; i++) { mma16816(s[i], qa[k], kb[2 * i], kb[2 * i + 1]); mma16816(s[i], ql[k], kb[2 * i], kb[2 * i + 1]); }
      }
#pragma unroll
      for (int i = 0; i < 2; i++)
#pragma unroll
        for (int e = 0; e < 2; e++)
          *reinterpret_cast<float2*>(&ss[(warp * 16 + g + 8 * e) * SP + j + 8 * i + c2]) = make_float2(s[i][2 * e], s[i][2 * e + 1]);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; i++) {      // softmax of two heads per warp
      const int r = 2 * warp + i;
      float x0 = 0.f, x1 = 0.f;
#pragma unroll
      for (int k = 0; k < 8; k++) {
        x0 += ss[(k * 16 + r) * SP + lane];
        if (KT > 32) x1 += ss[(k * 16 + r) * SP + lane + 32];
      }
      const int key = tile * KT + lane;
      x0 = key < n ? x0 * a.scale : -INFINITY;
      x1 = KT > 32 && key + 32 < n ? x1 * a.scale : -INFINITY;
      const float m = sml[2 * r], mn = fmaxf(m, warp_max(fmaxf(x0, x1)));      // finite: the first key of a tile is always seen
      const float p0 = __expf(x0 - mn), p1 = __expf(x1 - mn), f = __expf(m - mn);
      const float l = warp_sum(p0 + p1);
      const bf16 h0b = __float2bfloat16_rn(p0), h1b = __float2bfloat16_rn(p1);
      const int o0 = swz(r, lane, 64), o1 = swz(r, lane + 32, 64);
      ph[o0] = h0b; ph[16 * 64 + o0] = __float2bfloat16_rn(p0 - __bfloat162float(h0b));
      if (KT > 32) { ph[o1] = h1b; ph[16 * 64 + o1] = __float2bfloat16_rn(p1 - __bfloat162float(h1b)); }
      __syncwarp();
      if (lane == 0) { sal[r] = f; sml[2 * r] = mn; sml[2 * r + 1] = sml[2 * r + 1] * f + l; }
    }
    __syncthreads();
    const float f0 = sal[g], f1 = sal[g + 8];
#pragma unroll
    for (int j = 0; j < NP; j++)
#pragma unroll
      for (int i = 0; i < 2; i++) { o[j][i][0] *= f0; o[j][i][1] *= f0; o[j][i][2] *= f1; o[j][i][3] *= f1; }
    for (int k = 0; k < KT; k += 16) {
      uint32_t ah[4], al[4];
      const int at = swz(lane & 15, k + 8 * (lane >> 4), 64);
      ldsm4(ah, ph + at); ldsm4(al, ph + 16 * 64 + at);
#pragma unroll
      for (int j = 0; j < NP; j++) {
        const int c = (j * 8 + warp) * 16;
        if (c >= a.lp) continue;
        uint32_t vb[4];
        ldsm4t(vb, kt + swz(k + (lane & 15), c + 8 * (lane >> 4), width));
#pragma unroll
        for (int i = 0; i < 2; i++) { mma16816(o[j][i], ah, vb[2 * i], vb[2 * i + 1]); mma16816(o[j][i], al, vb[2 * i], vb[2 * i + 1]); }
      }
    }
  }
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 2; e++) {
    const int h = h0 + g + 8 * e;
    if (h >= a.heads) continue;
    float* dst = a.part + ((row * a.heads + h) * splits + sp) * (a.lp + 2);
    if (warp == 0 && (lane & 3) == 0) { dst[0] = sml[2 * (g + 8 * e)]; dst[1] = sml[2 * (g + 8 * e) + 1]; }
#pragma unroll
    for (int j = 0; j < NP; j++)
#pragma unroll
      for (int i = 0; i < 2; i++) {
        const int c = (j * 8 + warp) * 16 + 8 * i + c2;
        if (c < a.lp) *reinterpret_cast<float2*>(dst + 2 + c) = make_float2(o[j][i][2 * e], o[j][i][2 * e + 1]);
      }
  }
}

// grid (heads, rows): the splits of a head in order, normalised, as bf16 rows for the value up-projection.
__global__ void __launch_bounds__(1024) k_latent_combine(const LatentArgs a, int splits) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];
  float* ws = sm;                 // [splits]
  float* half1 = sm + splits;     // [lp]
  const int h = blockIdx.x, tid = threadIdx.x, lane = tid & 31, ldp = a.lp + 2;
  const long long row = blockIdx.y;
  const float* p = a.part + (row * a.heads + h) * (long long)splits * ldp;
  if (tid < 32) {
    float M = -INFINITY, L = 0.f;
    for (int s = lane; s < splits; s += 32) { const float m = p[(long long)s * ldp]; ws[s] = m; M = fmaxf(M, m); }
    M = warp_max(M);
    for (int s = lane; s < splits; s += 32) {
      const float w = ws[s] == -INFINITY ? 0.f : expf(ws[s] - M);
      L += w * p[(long long)s * ldp + 1];
      ws[s] = w;
    }
    L = 1.f / warp_sum(L);
    for (int s = lane; s < splits; s += 32) ws[s] *= L;
  }
  __syncthreads();
  const int part = tid >> 9, per = (splits + 1) / 2, s1 = min(splits, (part + 1) * per);
  for (int c0 = 0; c0 < a.lp; c0 += 512) {
    const int c = c0 + (tid & 511);
    float acc = 0.f;
    if (c < a.lp) {
#pragma unroll 8
      for (int s = part * per; s < s1; s++) acc = fmaf(ws[s], p[(long long)s * ldp + 2 + c], acc);   // an empty split holds zeros
      if (part) half1[c] = acc;
    }
    __syncthreads();
    if (!part && c < a.lp) reinterpret_cast<bf16*>(a.oc)[(row * a.heads + h) * a.lp + c] = __float2bfloat16_rn(acc + half1[c]);
  }
}

// grid (heads / 8, splits, rows): a block takes one contiguous range of the cached rows, staged 32 at a time in shared
// memory, each warp one head.  Partials (max, sum, unnormalised latent) go to part[row][head][split][lp + 2].
constexpr int LP_MAX = 32;   // kv_rank <= 1024
template <typename T, int PER>
__global__ void __launch_bounds__(256) k_latent_decode(const LatentArgs a, int splits) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];
  const int P = a.ld + 1;
  float* rows = sm;               // [32][P]
  float* qs = rows + 32 * P;      // [8][ld]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x * 8 + warp, sp = blockIdx.y;
  const long long row = blockIdx.z;
  const int b = (int)(row / a.T), t = (int)(row % a.T);
  const int n = a.first + t + 1, per = (n + splits - 1) / splits;
  const int kb = sp * per, ke = min(n, kb + per);
  const T* lat = reinterpret_cast<const T*>(a.latent) + (long long)b * a.maxT * a.ld;
  if (h < a.heads) for (int i = lane; i < a.ld; i += 32) qs[warp * a.ld + i] = a.qabs[(row * a.heads + h) * a.ld + i];
  float m = -INFINITY, l = 0.f, o[PER];
#pragma unroll
  for (int i = 0; i < PER; i++) o[i] = 0.f;
  for (int k0 = kb; k0 < ke; k0 += 32) {
    const int nk = min(32, ke - k0);
    __syncthreads();
    for (int i = threadIdx.x; i < nk * a.ld; i += 256) rows[(i / a.ld) * P + i % a.ld] = to_f<T>(lat[(long long)k0 * a.ld + i]);
    __syncthreads();
    if (h >= a.heads) continue;
    float s = -INFINITY;
    if (lane < nk) {
      s = 0.f;
      for (int i = 0; i < a.ld; i++) s = fmaf(qs[warp * a.ld + i], rows[lane * P + i], s);
      s *= a.scale;
    }
    const float mn = fmaxf(m, warp_max(s));
    const float p = expf(s - mn), f = expf(m - mn);
    l = l * f + warp_sum(p);
    m = mn;
#pragma unroll
    for (int i = 0; i < PER; i++) o[i] *= f;
    for (int k = 0; k < nk; k++) {
      const float pk = __shfl_sync(0xffffffffu, p, k);
#pragma unroll
      for (int i = 0; i < PER; i++)
        if (i * 32 + lane < a.lp) o[i] = fmaf(pk, rows[k * P + i * 32 + lane], o[i]);
    }
  }
  if (h >= a.heads) return;
  float* dst = a.part + ((row * a.heads + h) * splits + sp) * (a.lp + 2);
  if (lane == 0) { dst[0] = m; dst[1] = l; }
#pragma unroll
  for (int i = 0; i < PER; i++) if (i * 32 + lane < a.lp) dst[2 + i * 32 + lane] = o[i];
}

// grid (vdim / 32, heads, rows): combine the splits in order, then 32 rows of W_uv and the head's gate.
template <typename T>
__global__ void __launch_bounds__(1024) k_latent_decode_out(const LatentArgs a, int splits) {
  pdl_trigger();
  pdl_wait();
  constexpr int V = VecN<T>::n;
  extern __shared__ float sm[];
  float* oc = sm;                 // [lp], then [halves][lp] partial sums
  float* ws = oc + 2 * a.lp;      // [splits]
  __shared__ float total;
  const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tid = threadIdx.x;
  const long long row = blockIdx.z;
  const int ldp = a.lp + 2;
  const float* p = a.part + (row * a.heads + h) * (long long)splits * ldp;
  if (warp == 0) {
    float M = -INFINITY, L = 0.f;
    for (int s = lane; s < splits; s += 32) M = fmaxf(M, p[(long long)s * ldp]);
    M = warp_max(M);
    for (int s = lane; s < splits; s += 32) {
      const float ms = p[(long long)s * ldp], w = ms == -INFINITY ? 0.f : expf(ms - M);
      ws[s] = w;
      L += w * p[(long long)s * ldp + 1];
    }
    L = warp_sum(L);
    if (lane == 0) total = L;
  }
  __syncthreads();
  const int per = (splits + 1) / 2;
  for (int i = tid; i < 2 * a.lp; i += 1024) {
    const int c = i % a.lp, half = i / a.lp, s1 = min(splits, (half + 1) * per);
    float acc = 0.f;
#pragma unroll 8
    for (int s = half * per; s < s1; s++) acc = fmaf(ws[s], p[(long long)s * ldp + 2 + c], acc);   // an empty split holds zeros
    oc[i] = acc;
  }
  __syncthreads();
  const int e = blockIdx.x * 32 + warp;
  if (e >= a.vdim) return;
  const float g = to_f<T>(reinterpret_cast<const T*>(a.gate)[row * a.ld_gate + h]);
  const float f = 1.f / (total * (1.f + expf(-g)));
  const T* w = reinterpret_cast<const T*>(a.w_kv) + ((long long)a.heads * a.dim + (long long)h * a.vdim + e) * a.lp;
  float acc = 0.f;
#pragma unroll 2
  for (int c = lane * V; c < a.lp; c += 32 * V) {
    float x[V];
    load_vec<T, V>(w + c, x);
#pragma unroll
    for (int k = 0; k < V; k++) acc = fmaf(x[k], oc[c + k] + oc[a.lp + c + k], acc);
  }
  acc = warp_sum(acc);
  if (lane == 0) reinterpret_cast<T*>(a.o)[row * (long long)a.heads * a.vdim + (long long)h * a.vdim + e] = from_f<T>(acc * f);
}

// Opt-in to more than 48 KB of dynamic shared memory, once per kernel and device.
template <typename K> int allow_smem(K kernel, size_t bytes) {
  if (bytes > 227 * 1024) return femto_fail(FEMTO_ERR_UNSUPPORTED, "latent attention: a tile needs %zu bytes of shared memory", bytes);
  if (bytes > 48 * 1024) CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
  return 0;
}

}  // namespace

template <typename T> int latent_norms(const LatentArgs& a, cudaStream_t s) {
  CUDA_TRY(launch_dependent(k_latent_norms<T>, cdiv(2LL * a.B * a.T, 8), 256, 0, s, a));
  KERNEL_CHECK();
  return 0;
}
template int latent_norms<float>(const LatentArgs&, cudaStream_t);
template int latent_norms<bf16>(const LatentArgs&, cudaStream_t);

// A few new tokens per column: queries into the latent space, attention over the cached rows, back out.
static int latent_decode_tc(const LatentArgs& a, cudaStream_t s, bool& done) {
  const int N = a.first + a.T, rows = a.B * a.T, H = a.heads, hd = a.dim + a.rot_dim;
  const int width = round_up(a.ld, 64), nk = cdiv(width, 128), np = cdiv(a.lp, 128);
  auto bytes = [&](int kt) { return (size_t)2 * kt * width * 2 + 2 * 16 * 64 * 2 + 4 * (size_t)(8 * 16 * (kt + 4) + 48); };
  const int KT = bytes(64) <= 227 * 1024 ? 64 : 32;
  // the rotated queries (16 x rot_dim) pass through the space of the scores
  done = bytes(KT) <= 227 * 1024 && (hd & 7) == 0 && (a.dim & 7) == 0 && nk <= 9 && a.rot_dim <= 8 * (KT + 4);
  if (!done) return 0;
  const bf16* q = (const bf16*)a.q;
  for (int r0 = 0; r0 < rows; r0 += ROWS_STREAM) {      // qabs[row][head] = W_uk^T q
    RowsBatch bt;
    bt.x = hd; bt.w = (long long)a.lp * a.dp; bt.c = a.lp;
    FEMTO_TRY(rows_stream(q + (long long)r0 * H * hd, (long long)H * hd, (const bf16*)a.w_ukt, a.dp, a.qabs + (long long)r0 * H * a.lp, (long long)H * a.lp,
                          std::min(ROWS_STREAM, rows - r0), a.lp, a.dim, EPI_F32, H, bt, s));
  }
  const int tiles = cdiv(N, KT), blocks = cdiv(H, 16) * rows;
  int per = std::max(1, cdiv(tiles, std::max(1, device_sm_count() / blocks)));      // as many splits as fill the device once
  while ((size_t)rows * H * cdiv(tiles, per) * (a.lp + 2) > a.part_floats) per++;
  const int splits = cdiv(tiles, per);
#define LAUNCH(NK, NP) do { FEMTO_TRY(allow_smem(k_latent_decode_mma<NK, NP>, bytes(KT))); \
  CUDA_TRY(launch_dependent(k_latent_decode_mma<NK, NP>, dim3(cdiv(H, 16), splits, rows), 256, bytes(KT), s, a, splits, per, KT, width)); } while (0)
  if (nk <= 1) LAUNCH(1, 1);
  else if (nk <= 2) LAUNCH(2, 2);
  else if (nk <= 3) LAUNCH(3, 3);
  else if (nk <= 5 && np <= 4) LAUNCH(5, 4);
  else LAUNCH(9, 8);
#undef LAUNCH
  KERNEL_CHECK();
  CUDA_TRY(launch_dependent(k_latent_combine, dim3(H, rows), 1024, 4 * (size_t)(splits + a.lp), s, a, splits));
  KERNEL_CHECK();
  for (int r0 = 0; r0 < rows; r0 += ROWS_STREAM) {      // o[row][head] = W_uv oc sigmoid(gate)
    RowsBatch bt;
    bt.x = a.lp; bt.w = (long long)a.vdim * a.lp; bt.c = a.vdim;
    bt.gate = (const bf16*)a.gate + (long long)r0 * a.ld_gate; bt.ld_gate = a.ld_gate;
    FEMTO_TRY(rows_stream((const bf16*)a.oc + (long long)r0 * H * a.lp, (long long)H * a.lp, (const bf16*)a.w_kv + (long long)H * a.dim * a.lp, a.lp,
                          (bf16*)a.o + (long long)r0 * H * a.vdim, (long long)H * a.vdim, std::min(ROWS_STREAM, rows - r0), a.vdim, a.lp, EPI_STORE, H, bt, s));
  }
  return 0;
}

template <typename T> static int latent_decode(const LatentArgs& a, cudaStream_t s) {
  if constexpr (sizeof(T) == 2) {
    bool done = false;
    FEMTO_TRY(latent_decode_tc(a, s, done));
    if (done) return 0;
  }
  constexpr int V = VecN<T>::n;
  const int N = a.first + a.T, rows = a.B * a.T;
  const size_t absorb = 4 * (size_t)(a.dim + a.rot_dim + 1024 / (a.lp / V) * a.lp);
  FEMTO_TRY(allow_smem(k_absorb_q<T>, absorb));
  CUDA_TRY(launch_dependent(k_absorb_q<T>, dim3(a.heads, rows), 1024, absorb, s, a));
  KERNEL_CHECK();
  const int blocks = cdiv(a.heads, 8) * rows;
  int splits = std::max(1, std::min({LATENT_MAX_SPLITS, cdiv(N, 64), cdiv(2 * device_sm_count(), blocks)}));
  while (splits > 1 && (size_t)rows * a.heads * splits * (a.lp + 2) > a.part_floats) splits--;
  const size_t smem = 4 * (size_t)(32 * (a.ld + 1) + 8 * a.ld);
  const int per = cdiv(a.lp, 32);
  const dim3 grid(cdiv(a.heads, 8), splits, rows);
#define LAUNCH(PER) do { FEMTO_TRY(allow_smem(k_latent_decode<T, PER>, smem)); CUDA_TRY(launch_dependent(k_latent_decode<T, PER>, grid, 256, smem, s, a, splits)); } while (0)
  if (per <= 4) LAUNCH(4);
  else if (per <= 8) LAUNCH(8);
  else if (per <= 16) LAUNCH(16);
  else LAUNCH(32);
#undef LAUNCH
  KERNEL_CHECK();
  CUDA_TRY(launch_dependent(k_latent_decode_out<T>, dim3(cdiv(a.vdim, 32), a.heads, rows), 1024, 4 * (size_t)(2 * a.lp + splits), s, a, splits));
  KERNEL_CHECK();
  return 0;
}

template <typename T> int latent_attention(const LatentArgs& a, cudaStream_t s) {
  const int N = a.first + a.T, rows = a.B * a.T;
  if (a.vdim > 256 || a.dim + a.rot_dim > 512 || a.lp > 32 * LP_MAX)
    return femto_fail(FEMTO_ERR_UNSUPPORTED, "latent attention: dim %d + %d, vdim %d, rank %d", a.dim, a.rot_dim, a.vdim, a.kv_rank);
  if (a.T <= LATENT_FEW) return latent_decode<T>(a, s);
  if (a.rot_dims > 0) {
    if (a.rot_dims % 4 == 0 && a.dim % 2 == 0 && a.rot_dim % 2 == 0)
      CUDA_TRY(launch_dependent(k_rotate_q<T, 2>, cdiv((long long)rows * (a.rot_dims / 4), 256), 256, 0, s, a));
    else
      CUDA_TRY(launch_dependent(k_rotate_q<T, 1>, cdiv((long long)rows * (a.rot_dims / 2), 256), 256, 0, s, a));
    KERNEL_CHECK();
  }
  // keys and values of all N tokens of every column: [N][lp] x [heads (dim + vdim)][lp]^T
  const int wide = a.heads * (a.dim + a.vdim);
  GemmArgs g;
  g.ws = a.d->gemm_ws; g.ws_bytes = a.d->gemm_ws_bytes; g.status = a.d->status;
  g.A = a.latent; g.lda = a.ld; g.strideA = (long long)a.maxT * a.ld; g.B = a.w_kv; g.ldb = a.lp; g.strideB = 0;
  g.C = a.kv; g.ldc = wide; g.strideC = (long long)a.maxT * wide; g.M = N; g.N = wide; g.K = a.lp; g.epi = EPI_STORE; g.any_size = true;
  g.batch = a.B;
  FEMTO_TRY(gemm<T>(g, s));
  if (sizeof(T) == 2 && latent_attention_tc_supported(a)) return latent_attention_tc(a, s);
  const size_t smem = 4 * (size_t)((SQ + SK) * (a.dim + a.rot_dim + 1) + SK * a.vdim + SQ * (SK + 1) + 2 * SQ);
  FEMTO_TRY(allow_smem(k_latent_attn_simt<T>, smem));
  k_latent_attn_simt<T><<<dim3(cdiv(a.T, SQ), a.heads, a.B), 128, smem, s>>>(a, N);
  KERNEL_CHECK();
  return 0;
}
template int latent_attention<float>(const LatentArgs&, cudaStream_t);
template int latent_attention<bf16>(const LatentArgs&, cudaStream_t);

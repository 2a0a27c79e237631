// Attention over a cached low-rank latent: every token leaves one row [latent | rotated key part] that all heads share.
// A prompt expands the latents of its keys into per-head keys and values once and attends as usual; a few new tokens
// attend in the latent space instead, with queries taken through the key up-projection and the result through the value
// up-projection, so that a decode step reads each cached row once for all heads.
#include <algorithm>

#include "decoder.cuh"

namespace {

// ---- new rows: latent norm, rotations -------------------------------------------------------------------------------
// One warp per token row.
template <typename T>
__global__ void __launch_bounds__(256) k_latent_prep(const LatentArgs a) {
  pdl_trigger();
  const long long row = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (row >= (long long)a.B * a.T) return;
  const int lane = threadIdx.x & 31;
  const int b = (int)(row / a.T), t = (int)(row % a.T);
  const T* src = reinterpret_cast<const T*>(a.dkv) + row * a.ld_dkv;
  T* dst = reinterpret_cast<T*>(a.latent) + ((long long)b * a.maxT + a.first + t) * a.ld;
  float ss = 0.f;
  for (int c = lane; c < a.kv_rank; c += 32) { const float f = to_f<T>(src[c]); ss += f * f; }
  const float inv = 1.f / sqrtf(warp_sum(ss) / a.kv_rank + a.eps);
  for (int c = lane; c < a.kv_rank; c += 32) dst[c] = from_f<T>(to_f<T>(src[c]) * inv * a.dkv_norm[c]);
  const int half = a.rot_dims / 2, hd = a.dim + a.rot_dim;
  const float pos = (float)(a.first + t);
  src += a.kv_rank;
  dst += a.lp;
  T* q = reinterpret_cast<T*>(a.q) + row * (long long)a.heads * hd + a.dim;
  for (int i = lane; i < half; i += 32) {
    const float f = (float)pow(a.rot_base, -2.0 * i / a.rot_dims);
    float sn, cs;
    sincosf(pos * f, &sn, &cs);
    const float u = to_f<T>(src[i]), v = to_f<T>(src[i + half]);
    dst[i] = from_f<T>(u * cs - v * sn);
    dst[i + half] = from_f<T>(v * cs + u * sn);
    for (int h = 0; h < a.heads; h++) {
      T* qh = q + (long long)h * hd;
      const float qu = to_f<T>(qh[i]), qv = to_f<T>(qh[i + half]);
      qh[i] = from_f<T>(qu * cs - qv * sn);
      qh[i + half] = from_f<T>(qv * cs + qu * sn);
    }
  }
  for (int i = a.rot_dims + lane; i < a.rot_dim; i += 32) dst[i] = src[i];
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
// qabs[row][head] = [W_uk^T q (kv_rank), zeros up to lp, rotated q (rot_dim), zeros up to ld]
template <typename T>
__global__ void __launch_bounds__(256) k_absorb_q(const LatentArgs a) {
  pdl_trigger();
  extern __shared__ float qs[];
  const int h = blockIdx.y, hd = a.dim + a.rot_dim;
  const long long row = blockIdx.z;
  const T* q = reinterpret_cast<const T*>(a.q) + (row * a.heads + h) * hd;
  for (int i = threadIdx.x; i < hd; i += 256) qs[i] = to_f<T>(q[i]);
  __syncthreads();
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= a.ld) return;
  float acc = 0.f;
  if (c < a.kv_rank) {
    const T* w = reinterpret_cast<const T*>(a.w_kv) + (long long)h * a.dim * a.lp + c;
    for (int d = 0; d < a.dim; d++) acc = fmaf(qs[d], to_f<T>(w[(long long)d * a.lp]), acc);
  } else if (c >= a.lp && c < a.lp + a.rot_dim) {
    acc = qs[a.dim + c - a.lp];
  }
  a.qabs[(row * a.heads + h) * a.ld + c] = acc;
}

// grid (heads / 8, splits, rows): a block takes one contiguous range of the cached rows, staged 32 at a time in shared
// memory, each warp one head.  Partials (max, sum, unnormalised latent) go to part[row][head][split][lp + 2].
constexpr int LP_MAX = 32;   // kv_rank <= 1024
template <typename T, int PER>
__global__ void __launch_bounds__(256) k_latent_decode(const LatentArgs a, int splits) {
  pdl_trigger();
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

// grid (heads, rows): combine the splits in order, then W_uv and the head's gate.
template <typename T>
__global__ void __launch_bounds__(256) k_latent_decode_out(const LatentArgs a, int splits) {
  pdl_trigger();
  extern __shared__ float oc[];   // [lp]
  const int h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long row = blockIdx.y;
  const float* p = a.part + (row * a.heads + h) * (long long)splits * (a.lp + 2);
  float M = -INFINITY, L = 0.f;
  for (int s = 0; s < splits; s++) M = fmaxf(M, p[(long long)s * (a.lp + 2)]);
  for (int s = 0; s < splits; s++) {
    const float ms = p[(long long)s * (a.lp + 2)];
    if (ms != -INFINITY) L += p[(long long)s * (a.lp + 2) + 1] * expf(ms - M);
  }
  const float inv = 1.f / L;
  for (int c = threadIdx.x; c < a.lp; c += 256) {
    float acc = 0.f;
    for (int s = 0; s < splits; s++) {
      const float ms = p[(long long)s * (a.lp + 2)];
      if (ms != -INFINITY) acc += p[(long long)s * (a.lp + 2) + 2 + c] * expf(ms - M);
    }
    oc[c] = acc * inv;
  }
  __syncthreads();
  const float g = to_f<T>(reinterpret_cast<const T*>(a.gate)[row * a.ld_gate + h]);
  const float f = 1.f / (1.f + expf(-g));
  const T* w = reinterpret_cast<const T*>(a.w_kv) + (long long)(a.heads * a.dim + h * a.vdim) * a.lp;
  for (int e = warp; e < a.vdim; e += 8) {
    float acc = 0.f;
    for (int c = lane; c < a.kv_rank; c += 32) acc = fmaf(to_f<T>(w[(long long)e * a.lp + c]), oc[c], acc);
    acc = warp_sum(acc);
    if (lane == 0) reinterpret_cast<T*>(a.o)[row * (long long)a.heads * a.vdim + (long long)h * a.vdim + e] = from_f<T>(acc * f);
  }
}

// Opt-in to more than 48 KB of dynamic shared memory, once per kernel and device.
template <typename K> int allow_smem(K kernel, size_t bytes) {
  if (bytes > 227 * 1024) return femto_fail(FEMTO_ERR_UNSUPPORTED, "latent attention: a tile needs %zu bytes of shared memory", bytes);
  if (bytes > 48 * 1024) CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
  return 0;
}

}  // namespace

template <typename T> int latent_prep(const LatentArgs& a, cudaStream_t s) {
  k_latent_prep<T><<<cdiv((long long)a.B * a.T, 8), 256, 0, s>>>(a);
  KERNEL_CHECK();
  return 0;
}
template int latent_prep<float>(const LatentArgs&, cudaStream_t);
template int latent_prep<bf16>(const LatentArgs&, cudaStream_t);

template <typename T> int latent_attention(const LatentArgs& a, cudaStream_t s) {
  const int N = a.first + a.T, rows = a.B * a.T;
  if (a.vdim > 256 || a.dim + a.rot_dim > 512 || a.lp > 32 * LP_MAX)
    return femto_fail(FEMTO_ERR_UNSUPPORTED, "latent attention: dim %d + %d, vdim %d, rank %d", a.dim, a.rot_dim, a.vdim, a.kv_rank);
  if (a.T <= LATENT_FEW) {
    k_absorb_q<T><<<dim3(cdiv(a.ld, 256), a.heads, rows), 256, (a.dim + a.rot_dim) * 4, s>>>(a);
    KERNEL_CHECK();
    const int blocks = cdiv(a.heads, 8) * rows;
    int splits = std::max(1, std::min({LATENT_MAX_SPLITS, cdiv(N, 64), cdiv(2 * device_sm_count(), blocks)}));
    while (splits > 1 && (size_t)rows * a.heads * splits * (a.lp + 2) > a.part_floats) splits--;
    const size_t smem = 4 * (size_t)(32 * (a.ld + 1) + 8 * a.ld);
    const int per = cdiv(a.lp, 32);
    const dim3 grid(cdiv(a.heads, 8), splits, rows);
#define LAUNCH(PER) do { FEMTO_TRY(allow_smem(k_latent_decode<T, PER>, smem)); k_latent_decode<T, PER><<<grid, 256, smem, s>>>(a, splits); } while (0)
    if (per <= 4) LAUNCH(4);
    else if (per <= 8) LAUNCH(8);
    else if (per <= 16) LAUNCH(16);
    else LAUNCH(32);
#undef LAUNCH
    KERNEL_CHECK();
    k_latent_decode_out<T><<<dim3(a.heads, rows), 256, a.lp * 4, s>>>(a, splits);
    KERNEL_CHECK();
    return 0;
  }
  // keys and values of all N tokens of every column: [N][lp] x [heads (dim + vdim)][lp]^T
  const int wide = a.heads * (a.dim + a.vdim);
  GemmArgs g;
  g.ws = a.d->gemm_ws; g.ws_bytes = a.d->gemm_ws_bytes; g.status = a.d->status;
  g.A = a.latent; g.lda = a.ld; g.strideA = (long long)a.maxT * a.ld; g.B = a.w_kv; g.ldb = a.lp; g.strideB = 0;
  g.C = a.kv; g.ldc = wide; g.strideC = (long long)a.maxT * wide; g.M = N; g.N = wide; g.K = a.lp; g.epi = EPI_STORE;
  for (int b = 0; b < a.B; b++) {
    FEMTO_TRY(gemm<T>(g, s));
    g.A = reinterpret_cast<const T*>(g.A) + g.strideA;
    g.C = reinterpret_cast<T*>(g.C) + g.strideC;
  }
  if (sizeof(T) == 2 && latent_attention_tc_supported(a)) return latent_attention_tc(a, s);
  const size_t smem = 4 * (size_t)((SQ + SK) * (a.dim + a.rot_dim + 1) + SK * a.vdim + SQ * (SK + 1) + 2 * SQ);
  FEMTO_TRY(allow_smem(k_latent_attn_simt<T>, smem));
  k_latent_attn_simt<T><<<dim3(cdiv(a.T, SQ), a.heads, a.B), 128, smem, s>>>(a, N);
  KERNEL_CHECK();
  return 0;
}
template int latent_attention<float>(const LatentArgs&, cudaStream_t);
template int latent_attention<bf16>(const LatentArgs&, cudaStream_t);

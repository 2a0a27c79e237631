// Recurrent token mixers with an fp32 matrix state per head: a decayed sum of outer products (lightning attention) and
// the gated delta rule with one decay per key channel.  The state is kept as [vdim][dim]: its vdim columns are independent
// recurrences that share q, k and the decays, so a block owns 32 of them, eight lanes each, for any number of tokens.
#include "decoder.cuh"

namespace {

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
// log(1 + e^z) without overflow or cancellation
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

template <int NI> struct Tile { static constexpr int TOK = NI >= 8 ? 8 : 16; };   // tokens staged at a time

// q / k / g of one head, v of this block's 32 columns and beta for `n` tokens from row `r0` into shared memory.
template <typename T, bool DELTA, int NI>
__global__ void __launch_bounds__(256) k_recurrence(const RecurrenceArgs a) {
  pdl_trigger();
  pdl_wait();
  constexpr int DP = 32 * NI, TT = Tile<NI>::TOK;
  __shared__ __align__(16) float sq[TT][DP], sk[TT][DP], sg[DELTA ? TT : 1][DELTA ? DP : 4], sv[TT][32], sb[TT];
  const int h = blockIdx.y, b = blockIdx.z;
  const int lane = threadIdx.x & 31, sub = lane & 7, colb = (threadIdx.x >> 5) * 4 + (lane >> 3);
  const int e = blockIdx.x * 32 + colb;
  const int qh = h / (a.heads / a.qk_heads);
  const int D = a.dim, E = a.vdim;
  float* Sp = a.S + (((long long)b * a.heads + h) * E + min(e, E - 1)) * D;
  float s[NI * 4];
#pragma unroll
  for (int i = 0; i < NI; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int d = 4 * (sub + 8 * i) + j;
      s[i * 4 + j] = (e < E && d < D) ? Sp[d] : 0.f;
    }
  const float decay = DELTA ? 1.f : a.decay[h];
  for (int t0 = 0; t0 < a.T; t0 += TT) {
    const int n = min(TT, a.T - t0);
    const long long r0 = (long long)b * a.T + t0;
    __syncthreads();
    for (int i = threadIdx.x; i < n * DP; i += 256) {
      const int t = i / DP, d = i % DP;
      float q = 0.f, k = 0.f;
      if (d < D) {
        const long long iq = (r0 + t) * a.ldq + (long long)qh * D + d, ik = (r0 + t) * a.ldk + (long long)qh * D + d;
        if (DELTA) {
          q = reinterpret_cast<const float*>(a.q)[iq]; k = reinterpret_cast<const float*>(a.k)[ik];
        } else {
          q = silu_f(to_f<T>(reinterpret_cast<const T*>(a.q)[iq])); k = silu_f(to_f<T>(reinterpret_cast<const T*>(a.k)[ik]));
        }
      }
      sq[t][d] = q; sk[t][d] = k;
      if (DELTA) sg[t][d] = d < D ? a.g[(r0 + t) * ((long long)a.heads * D) + (long long)h * D + d] : 0.f;
    }
    for (int i = threadIdx.x; i < n * 32; i += 256) {
      const int t = i / 32, c = blockIdx.x * 32 + i % 32;
      float v = c < E ? to_f<T>(reinterpret_cast<const T*>(a.v)[(r0 + t) * a.ldv + (long long)h * E + c]) : 0.f;
      if (!DELTA) v = silu_f(v);
      sv[t][i % 32] = v;
    }
    if (DELTA && threadIdx.x < n) sb[threadIdx.x] = a.beta[(r0 + threadIdx.x) * a.heads + h];
    __syncthreads();
    for (int t = 0; t < n; t++) {
      float o = 0.f;
      if constexpr (DELTA) {
        float dot = 0.f;
#pragma unroll
        for (int i = 0; i < NI; i++) {
          const float4 g = *reinterpret_cast<const float4*>(&sg[t][4 * (sub + 8 * i)]), k = *reinterpret_cast<const float4*>(&sk[t][4 * (sub + 8 * i)]);
          s[i * 4] *= g.x; s[i * 4 + 1] *= g.y; s[i * 4 + 2] *= g.z; s[i * 4 + 3] *= g.w;
          dot += s[i * 4] * k.x; dot += s[i * 4 + 1] * k.y; dot += s[i * 4 + 2] * k.z; dot += s[i * 4 + 3] * k.w;
        }
        dot += __shfl_xor_sync(0xffffffffu, dot, 1); dot += __shfl_xor_sync(0xffffffffu, dot, 2); dot += __shfl_xor_sync(0xffffffffu, dot, 4);
        const float u = sb[t] * (sv[t][colb] - dot);
#pragma unroll
        for (int i = 0; i < NI; i++) {
          const float4 k = *reinterpret_cast<const float4*>(&sk[t][4 * (sub + 8 * i)]), q = *reinterpret_cast<const float4*>(&sq[t][4 * (sub + 8 * i)]);
          s[i * 4] += k.x * u; s[i * 4 + 1] += k.y * u; s[i * 4 + 2] += k.z * u; s[i * 4 + 3] += k.w * u;
          o += s[i * 4] * q.x; o += s[i * 4 + 1] * q.y; o += s[i * 4 + 2] * q.z; o += s[i * 4 + 3] * q.w;
        }
      } else {
        const float u = sv[t][colb];
#pragma unroll
        for (int i = 0; i < NI; i++) {
          const float4 k = *reinterpret_cast<const float4*>(&sk[t][4 * (sub + 8 * i)]), q = *reinterpret_cast<const float4*>(&sq[t][4 * (sub + 8 * i)]);
          s[i * 4] = decay * s[i * 4] + k.x * u; s[i * 4 + 1] = decay * s[i * 4 + 1] + k.y * u;
          s[i * 4 + 2] = decay * s[i * 4 + 2] + k.z * u; s[i * 4 + 3] = decay * s[i * 4 + 3] + k.w * u;
          o += s[i * 4] * q.x; o += s[i * 4 + 1] * q.y; o += s[i * 4 + 2] * q.z; o += s[i * 4 + 3] * q.w;
        }
      }
      o += __shfl_xor_sync(0xffffffffu, o, 1); o += __shfl_xor_sync(0xffffffffu, o, 2); o += __shfl_xor_sync(0xffffffffu, o, 4);
      if (sub == 0 && e < E) reinterpret_cast<T*>(a.o)[(r0 + t) * ((long long)a.heads * E) + (long long)h * E + e] = from_f<T>(o);
    }
  }
#pragma unroll
  for (int i = 0; i < NI; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int d = 4 * (sub + 8 * i) + j;
      if (e < E && d < D) Sp[d] = s[i * 4 + j];
    }
}

// Input x[t - back] of channel c: from this call's rows, or from the inputs kept of earlier calls (zeros before the start).
template <typename T>
__device__ __forceinline__ float conv_input(const DeltaPrepArgs& a, int b, int t, int back, int seg, int c, int chan, int channels) {
  const int r = t - back;
  if (r >= 0) return to_f<T>(reinterpret_cast<const T*>(a.proj)[((long long)b * a.T + r) * a.ldp + seg + c]);
  return to_f<T>(reinterpret_cast<const T*>(a.tail_in)[((long long)b * (a.taps - 1) + (a.taps - 1 + r)) * channels + chan]);
}

// One warp per unit: q head, k head (convolution, silu, unit vector), v head (convolution, silu), or the decays of a head.
template <typename T>
__global__ void __launch_bounds__(256) k_delta_prep(const DeltaPrepArgs a) {
  pdl_trigger();
  pdl_wait();
  const int units = 2 * a.kv_heads + 2 * a.heads;
  const long long it = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (it >= (long long)a.B * a.T * units) return;
  const int lane = threadIdx.x & 31;
  const long long row = it / units;
  int u = (int)(it % units);
  const int b = (int)(row / a.T), t = (int)(row % a.T);
  const int G = a.kv_heads, H = a.heads, D = a.dim, E = a.vdim, n = a.taps;
  const int channels = 2 * G * D + H * E;
  if (u < 2 * G + H) {
    const bool is_q = u < G, is_v = u >= 2 * G;
    const int head = is_q ? u : is_v ? u - 2 * G : u - G, size = is_v ? E : D;
    const int seg = is_q ? a.s_q : is_v ? a.s_v : a.s_k;
    const int chan0 = is_q ? 0 : is_v ? 2 * G * D : G * D;
    const float* taps = is_q ? a.conv_q : is_v ? a.conv_v : a.conv_k;
    float ss = 0.f;
    float y[8];                      // sizes up to 256
#pragma unroll
    for (int i = 0; i < 8; i++) {
      const int c = head * size + i * 32 + lane;
      y[i] = 0.f;
      if (i * 32 + lane < size) {
        float acc = 0.f;
        for (int j = 0; j < n; j++) acc += taps[(long long)c * n + j] * conv_input<T>(a, b, t, n - 1 - j, seg, c, chan0 + c, channels);
        y[i] = silu_f(acc);
        ss += y[i] * y[i];
      }
    }
    float f = 1.f;
    if (!is_v) {
      f = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
      if (is_q) f *= 1.f / sqrtf((float)D);
    }
#pragma unroll
    for (int i = 0; i < 8; i++) {
      const int c = i * 32 + lane;
      if (c < size) {
        if (is_v) reinterpret_cast<T*>(a.vv)[row * H * E + (long long)head * E + c] = from_f<T>(y[i]);
        else (is_q ? a.qn : a.kn)[row * G * D + (long long)head * D + c] = y[i] * f;
      }
    }
  } else {
    const int head = u - 2 * G - H;
    const float rate = expf(a.a_log[head]);
    for (int c = lane; c < D; c += 32) {
      const long long i = row * H * D + (long long)head * D + c;
      a.gd[i] = expf(-rate * softplus_f(a.gd[i] + a.dt_bias[head * D + c]));
    }
    if (lane == 0) {
      const float z = to_f<T>(reinterpret_cast<const T*>(a.proj)[row * a.ldp + a.s_b + head]);
      a.beta[row * H + head] = 1.f / (1.f + expf(-z));
    }
  }
}

// The last taps - 1 inputs of every convolution after this call's rows.
template <typename T>
__global__ void __launch_bounds__(256) k_conv_tail(const DeltaPrepArgs a) {
  pdl_trigger();
  pdl_wait();
  const int G = a.kv_heads, D = a.dim, channels = 2 * G * D + a.heads * a.vdim, keep = a.taps - 1;
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= (long long)a.B * keep * channels) return;
  const int chan = (int)(i % channels), k = (int)(i / channels % keep), b = (int)(i / channels / keep);
  const int seg = chan < G * D ? a.s_q + chan : chan < 2 * G * D ? a.s_k + chan - G * D : a.s_v + chan - 2 * G * D;
  const int r = a.T - keep + k;
  reinterpret_cast<T*>(a.tail_out)[i] = r >= 0 ? reinterpret_cast<const T*>(a.proj)[((long long)b * a.T + r) * a.ldp + seg]
                                               : reinterpret_cast<const T*>(a.tail_in)[((long long)b * keep + keep + r) * channels + chan];
}

// ---- one token -----------------------------------------------------------------------------------------------------------
// The whole mixer between the packed projection and the output projection for one new token: convolutions, unit vectors,
// both low-rank projections, state update, read-out, norm and gate.  One block per (head, column).
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

template <typename T> __device__ __forceinline__ float row_dot(const T* __restrict__ w, const float* x, int n, int lane) {
  constexpr int V = VecN<T>::n;      // rows are padded to multiples of 8 with zeros
  float acc = 0.f;
  for (int c = lane * V; c < n; c += 32 * V) {
    float f[V];
    load_vec<T, V>(w + c, f);
#pragma unroll
    for (int e = 0; e < V; e++) acc = fmaf(f[e], x[c + e], acc);
  }
  return warp_sum(acc);
}

template <typename T, int NI>
__global__ void __launch_bounds__(1024) k_delta_decode(const DeltaDecodeArgs a) {
  pdl_trigger();
  pdl_wait();
  constexpr int DP = 32 * NI;
  const DeltaPrepArgs& p = a.p;
  extern __shared__ __align__(16) float sm[];
  float *sq = sm, *sk = sq + DP, *sg = sk + DP, *sv = sg + DP, *so = sv + p.vdim, *sz = so + p.vdim, *sa = sz + p.vdim, *sb = sa + a.ra;
  __shared__ float red[32], f_q, f_k;
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int H = p.heads, G = p.kv_heads, D = p.dim, E = p.vdim, n = p.taps, keep = n - 1;
  const int qh = h / (H / G), channels = 2 * G * D + H * E;
  const T* proj = reinterpret_cast<const T*>(p.proj) + (long long)b * p.ldp;
  const T* tin = reinterpret_cast<const T*>(p.tail_in) + (long long)b * keep * channels;
  T* tout = reinterpret_cast<T*>(p.tail_out) + (long long)b * keep * channels;
  for (int i = tid; i < a.ra; i += 1024) sa[i] = to_f<T>(proj[a.s_a1 + i]);
  for (int i = tid; i < a.rg; i += 1024) sb[i] = to_f<T>(proj[a.s_g1 + i]);
  for (int i = tid; i < 2 * DP + E; i += 1024) {
    const int which = i < DP ? 0 : i < 2 * DP ? 1 : 2, c = which == 2 ? i - 2 * DP : i - which * DP;
    const int size = which == 2 ? E : D, head = which == 2 ? h : qh;
    float y = 0.f;
    if (c < size) {
      const int at = head * size + c, chan = (which == 0 ? 0 : which == 1 ? G * D : 2 * G * D) + at;
      const float* taps = (which == 0 ? p.conv_q : which == 1 ? p.conv_k : p.conv_v) + (long long)at * n;
      const T now = proj[(which == 0 ? p.s_q : which == 1 ? p.s_k : p.s_v) + at];
      const bool writes = which == 2 || h % (H / G) == 0;      // the heads of a group share q and k
      float acc = 0.f;
      for (int j0 = 0; j0 < keep; j0 += 4) {          // four loads in flight before the first store
        T x[4];
#pragma unroll
        for (int j = 0; j < 4; j++) if (j0 + j < keep) x[j] = tin[(long long)(j0 + j) * channels + chan];
#pragma unroll
        for (int j = 0; j < 4; j++)
          if (j0 + j < keep) {
            acc = fmaf(taps[j0 + j], to_f<T>(x[j]), acc);
            if (writes && j0 + j > 0) tout[(long long)(j0 + j - 1) * channels + chan] = x[j];
          }
      }
      if (writes && keep > 0) tout[(long long)(keep - 1) * channels + chan] = now;
      y = silu_f(fmaf(taps[keep], to_f<T>(now), acc));
      if (which == 2) y = round_to<T>(y);
    }
    (which == 0 ? sq : which == 1 ? sk : sv)[c] = y;
  }
  __syncthreads();
  if (warp < 2) {
    const float* x = warp ? sk : sq;
    float ss = 0.f;
    for (int c = lane; c < D; c += 32) ss += x[c] * x[c];
    ss = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
    if (lane == 0) { if (warp) f_k = ss; else f_q = ss * (1.f / sqrtf((float)D)); }
  }
  const float rate = expf(p.a_log[h]);
#pragma unroll 4
  for (int i = warp; i < D + E; i += 32) {
    const bool decay = i < D;
    const int c = decay ? i : i - D, r = decay ? a.ra : a.rg;
    const T* w = reinterpret_cast<const T*>(decay ? a.w_a2 : a.w_g2) + (long long)(h * (decay ? D : E) + c) * r;
    const float z = row_dot<T>(w, decay ? sa : sb, r, lane);
    if (lane == 0) (decay ? sg : sz)[c] = z;
  }
  __syncthreads();
  for (int i = tid; i < DP + E; i += 1024) {
    if (i < DP) sg[i] = i < D ? expf(-rate * softplus_f(sg[i] + p.dt_bias[h * D + i])) : 0.f;
    else sz[i - DP] = sigmoid_f(round_to<T>(sz[i - DP]));
  }
  __syncthreads();
  const float beta = sigmoid_f(to_f<T>(proj[p.s_b + h])), fk = f_k, fq = f_q;
  const int sub = tid & 7;
  const bool vec = (D & 3) == 0;
  for (int e = tid >> 3; e < (E + 127) / 128 * 128; e += 128) {
    float* Sp = a.S + (((long long)b * H + h) * E + min(e, E - 1)) * D;
    float s[NI][4], dot = 0.f;
#pragma unroll
    for (int i = 0; i < NI; i++) {
      const int d = 4 * (sub + 8 * i);
      if (vec) {
        const float4 v = d < D && e < E ? *reinterpret_cast<const float4*>(Sp + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        s[i][0] = v.x; s[i][1] = v.y; s[i][2] = v.z; s[i][3] = v.w;
      } else {
#pragma unroll
        for (int j = 0; j < 4; j++) s[i][j] = d + j < D && e < E ? Sp[d + j] : 0.f;
      }
    }
#pragma unroll
    for (int i = 0; i < NI; i++)
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const int d = 4 * (sub + 8 * i) + j;
        s[i][j] *= sg[d];
        dot = fmaf(s[i][j], sk[d] * fk, dot);
      }
    dot += __shfl_xor_sync(0xffffffffu, dot, 1); dot += __shfl_xor_sync(0xffffffffu, dot, 2); dot += __shfl_xor_sync(0xffffffffu, dot, 4);
    const float u = beta * ((e < E ? sv[e] : 0.f) - dot);
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < NI; i++)
#pragma unroll
      for (int j = 0; j < 4; j++) {
        const int d = 4 * (sub + 8 * i) + j;
        s[i][j] = fmaf(sk[d] * fk, u, s[i][j]);
        o = fmaf(s[i][j], sq[d] * fq, o);
      }
    o += __shfl_xor_sync(0xffffffffu, o, 1); o += __shfl_xor_sync(0xffffffffu, o, 2); o += __shfl_xor_sync(0xffffffffu, o, 4);
    if (e < E) {
#pragma unroll
      for (int i = 0; i < NI; i++) {
        const int d = 4 * (sub + 8 * i);
        if (vec) {
          if (d < D) *reinterpret_cast<float4*>(Sp + d) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; j++) if (d + j < D) Sp[d + j] = s[i][j];
        }
      }
      if (sub == 0) so[e] = round_to<T>(o);
    }
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < E; c += 1024) ss += so[c] * so[c];
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = warp_sum(red[lane]);
  const float inv = 1.f / sqrtf(ss / E + a.eps);
  T* out = reinterpret_cast<T*>(a.out) + ((long long)b * H + h) * E;
  for (int c = tid; c < E; c += 1024) out[c] = from_f<T>(so[c] * inv * a.norm[c] * sz[c]);
}

}  // namespace

template <typename T> int recurrence(const RecurrenceArgs& a, cudaStream_t s) {
  const dim3 grid(cdiv(a.vdim, 32), a.heads, a.B);
  const bool delta = a.beta != nullptr;
#define LAUNCH(NI) if (delta) CUDA_TRY(launch_dependent(k_recurrence<T, true, NI>, grid, 256, 0, s, a)); else CUDA_TRY(launch_dependent(k_recurrence<T, false, NI>, grid, 256, 0, s, a))
  if (a.dim <= 32) { LAUNCH(1); }
  else if (a.dim <= 64) { LAUNCH(2); }
  else if (a.dim <= 128) { LAUNCH(4); }
  else if (a.dim <= 256) { LAUNCH(8); }
  else return femto_fail(FEMTO_ERR_UNSUPPORTED, "recurrence: dim %d > 256", a.dim);
#undef LAUNCH
  KERNEL_CHECK();
  return 0;
}
template int recurrence<float>(const RecurrenceArgs&, cudaStream_t);
template int recurrence<bf16>(const RecurrenceArgs&, cudaStream_t);

template <typename T> int conv_tail(const DeltaPrepArgs& a, cudaStream_t s) {
  if (a.taps <= 1) return 0;
  const long long m = (long long)a.B * (a.taps - 1) * (2 * a.kv_heads * a.dim + a.heads * a.vdim);
  CUDA_TRY(launch_dependent(k_conv_tail<T>, cdiv(m, 256), 256, 0, s, a));
  KERNEL_CHECK();
  return 0;
}
template int conv_tail<float>(const DeltaPrepArgs&, cudaStream_t);
template int conv_tail<bf16>(const DeltaPrepArgs&, cudaStream_t);

template <typename T> int delta_prep(const DeltaPrepArgs& a, cudaStream_t s) {
  if (a.dim > 256 || a.vdim > 256) return femto_fail(FEMTO_ERR_UNSUPPORTED, "delta rule: dim %d / vdim %d > 256", a.dim, a.vdim);
  const long long n = (long long)a.B * a.T * (2 * a.kv_heads + 2 * a.heads);
  CUDA_TRY(launch_dependent(k_delta_prep<T>, cdiv(n, 8), 256, 0, s, a));
  KERNEL_CHECK();
  return conv_tail<T>(a, s);
}
template int delta_prep<float>(const DeltaPrepArgs&, cudaStream_t);
template int delta_prep<bf16>(const DeltaPrepArgs&, cudaStream_t);

template <typename T> int delta_decode(const DeltaDecodeArgs& a, cudaStream_t s) {
  const dim3 grid(a.p.heads, a.p.B);
  const int ni = a.p.dim <= 32 ? 1 : a.p.dim <= 64 ? 2 : a.p.dim <= 128 ? 4 : 8;
  if (a.p.dim > 256 || a.p.vdim > 256) return femto_fail(FEMTO_ERR_UNSUPPORTED, "delta rule: dim %d / vdim %d > 256", a.p.dim, a.p.vdim);
  const size_t smem = 4 * (size_t)(3 * 32 * ni + 3 * a.p.vdim + a.ra + a.rg);
  if (smem > 48 * 1024) return femto_fail(FEMTO_ERR_UNSUPPORTED, "delta rule: ranks %d and %d are too large", a.ra, a.rg);
#define LAUNCH(NI) CUDA_TRY(launch_dependent(k_delta_decode<T, NI>, grid, 1024, smem, s, a))
  if (ni == 1) LAUNCH(1);
  else if (ni == 2) LAUNCH(2);
  else if (ni == 4) LAUNCH(4);
  else LAUNCH(8);
#undef LAUNCH
  KERNEL_CHECK();
  return 0;
}
template int delta_decode<float>(const DeltaDecodeArgs&, cudaStream_t);
template int delta_decode<bf16>(const DeltaDecodeArgs&, cudaStream_t);

// Decoders given as a list of layers (include/femto.h: femto_decoder_*): derived sizes, packed weights and workspace,
// and the mixers' entry points.  Inference only; the state that outlives a call is in the cache (kv_cache.cuh).
#pragma once
#include <string>
#include <vector>

#include "kv_cache.cuh"

static inline int round_up(int n, int k) { return (n + k - 1) / k * k; }

// The packed input projection of a mixer is ONE product: its segments follow each other in the columns of a row of
// `proj`, every segment starting at a multiple of 8 (16-byte loads, TMA operands); the gaps come from zero weights.
struct DecLayer {
  femto_layer_config c;
  int own = 0;                        // layer that holds the tensors
  std::vector<float> decay;
  float* decay_dev = nullptr;
  std::vector<float> freq;            // latent attention: rot_base^(-2i/rot_dims)
  float* freq_dev = nullptr;
  // element offsets into Theta of what is read there in fp32
  long long norm1 = -1, norm1b = -1, norm2 = -1, norm2b = -1, mix_norm = -1, conv_q = -1, conv_k = -1, conv_v = -1,
            a_log = -1, dt_bias = -1, dq_norm = -1, dkv_norm = -1, q_norm = -1, k_norm = -1, sink = -1, q_bias = -1, k_bias = -1, v_bias = -1,
            lq1 = -1, lk1 = -1, lq2 = -1, lk2 = -1, router_bias = -1;
  // packed compute-type weights, row-major [out][in]
  void *w_in = nullptr, *w_o = nullptr, *w_a2 = nullptr, *w_g2 = nullptr, *w_uq = nullptr, *w_kv = nullptr, *w_ukt = nullptr, *w_gu = nullptr,
       *w_down = nullptr, *w_router = nullptr;      // experts: w_gu [experts][ffp][width] (up), w_down [experts][width][ffp]
  int n_in = 0;                       // columns of proj
  int n_kv = 0, vo = 0;               // attention: columns of a cached row, which follow those of proj in w_in; where the values start
  int kv_layer = 0;                   // attention: layer whose cache holds the keys and values
  float *bias = nullptr, *lambda = nullptr;   // attention: [n_in + n_kv]; one number
  int s_q = 0, s_k = 0, s_v = 0, s_g = 0, s_b = 0, s_a1 = 0, s_g1 = 0, s_dkv = 0;   // segment starts
  int ra = 0, rg = 0;                 // decay_rank / gate_rank rounded up to 8
  int qp = 0, lp = 0, ld = 0, dp = 0; // q_rank, kv_rank rounded up to 8; pitch of a cached latent row; dim rounded up to 8
  int ffp = 0;                        // ff rounded up to 32 (experts: to 8): the feed-forward's products are this wide
  int qk_heads() const { return c.mixer == FEMTO_MIXER_CHANNEL_DELTA ? c.kv_heads : c.heads; }
};

struct DecoderStack {
  femto_decoder_config cfg;
  std::vector<DecLayer> layers;
  std::vector<femto_decoder_tensor> tensors;
  std::vector<femto_layer_config> layer_cfg;
  long long nparams = 0, off_embed = 0, off_final = 0;
  bool bf = false, weights_valid = false;
  char* arena = nullptr;
  unsigned int* status = nullptr;
  void* embed = nullptr;              // [vocab][width] compute type: input table
  void* head = nullptr;               // output head (the same table when tied)
  // workspace of one internal pass of up to max_rows tokens
  int* tok0 = nullptr;
  int* want = nullptr;                // [max_rows]
  float* x = nullptr;                 // residual stream, fp32
  void *hn = nullptr, *hn2 = nullptr, *y = nullptr, *y2 = nullptr, *proj = nullptr, *mixo = nullptr, *mixg = nullptr, *gu = nullptr, *act = nullptr;
  float *qn = nullptr, *kn = nullptr, *gd = nullptr, *beta = nullptr;
  void *vv = nullptr, *g2 = nullptr, *cq = nullptr, *q = nullptr;
  float* qabs = nullptr;              // latent attention, few rows: queries in the latent space
  void* oc = nullptr;                 // and results there
  // experts: router logits, choices, places, counts, runs, lists of a few rows' choices; sorted inputs and results
  float *moe_z = nullptr, *moe_weight = nullptr;
  int *moe_expert = nullptr, *moe_slot = nullptr, *moe_counts = nullptr, *moe_groups = nullptr, *moe_lists = nullptr;
  void *moe_x = nullptr, *moe_act = nullptr, *moe_out = nullptr;
  char* chunk_ws = nullptr;           // chunked recurrences: operands of the chunks of one segment
  size_t chunk_ws_bytes = 0;
  void* gemm_ws = nullptr;
  size_t gemm_ws_bytes = 0;
};

int decoder_fill(DecoderStack* d, const femto_decoder_config* cfg);
int decoder_create(const femto_decoder_config* cfg, femto_handle** out);
void decoder_free(DecoderStack* d);
int decoder_refresh(femto_handle* h, const float* theta, cudaStream_t s);
int decoder_step(femto_handle* h, femto_kv_cache* c, const float* theta, const int* tokens, int B, int T, const int* h_want,
                 int n_want, float* logits_out, float* residuals_out, cudaStream_t s);
int decoder_cache_create(femto_handle* h, int max_batch, int max_len, femto_kv_cache** out);
int decoder_cache_reset(femto_kv_cache* c, cudaStream_t s);

// ---- streaming kernels (decoder_stream.cu) ------------------------------------------------------------------------
// What the experts made of a row: out[slot ? slot[p] : p] for the pairs p = row * top + k, with their weights.
struct MoeRows {
  const void* out = nullptr;
  const int* slot = nullptr;
  const float* weight = nullptr;
  int top = 0;
};
// The norms that follow a sum: h = rms_norm(x) w and, with h2, h2 = rms_norm(x) w2 (h may be NULL: none)
template <typename T> struct NextNorms { const float* w = nullptr; T* h = nullptr; const float* w2 = nullptr; T* h2 = nullptr; };
template <typename T> struct DecStream {
  // x = scale * table[token] (fp32), then the norms
  static int embed(const T* table, const int* tokens, int ld_tok, int B, int T_, int base, int vocab, float scale, float* x,
                   const NextNorms<T>& n, int d, float eps, unsigned int* status, cudaStream_t s);
  // x += y + (y2, or the weighted sum of the experts' rows, or nothing), then the norms
  static int parallel_resid(float* x, const T* y, const T* y2, const MoeRows& m, const NextNorms<T>& n, int rows, int d, float eps,
                            cudaStream_t s);
  // x += m rms_norm(y) w_post;  h = rms_norm(x) w_pre (skipped when h is NULL)
  static int resid_norm(float* x, const T* y, const float* w_post, float m, const float* w_pre, T* h, int rows, int d, float eps,
                        cudaStream_t s);
  // h[i] = rms_norm(x[row i]) w, row i = want ? want[i] : (i + 1) stride - 1
  static int gather_norm(const float* x, const int* want, int stride, const float* w, T* h, int n, int d, float eps,
                         cudaStream_t s);
  // out[r][g] = rms_norm over each of `groups` runs of `size` of in[r], times w (size, or groups*size when w_all), times sigmoid(gate)
  static int gated_norm(const T* in, const float* w, bool w_all, const T* gate, long long ldg, T* out, int rows, int groups, int size,
                        float eps, cudaStream_t s);
  // act[r][j] = silu(gate) * up from rows of interleaved groups of 32 gate and 32 up columns
  static int gated_mlp(const T* gu, T* act, int rows, int ffp, cudaStream_t s);
};
// weight packing: dst[(r / group) * step + r % group + dst_row][c] = src[r][c], c < cols (dst pitch ldd)
template <typename T>
int pack_transposed(const float* src, int batch, int rows, int cols, T* dst, int ld_rows, int ld_cols, cudaStream_t s);   // dst[b][c][r] = src[b][r][c]
template <typename T>
int pack_rows(const float* src, int rows, int cols, T* dst, long long ldd, int dst_row, int group, int step, cudaStream_t s);

// ---- products -------------------------------------------------------------------------------------------------------
// C[M][N] = X[M][K] W[N][K]^T; epi EPI_STORE (compute type), EPI_F32, or EPI_SWIGLU (W holds 2 N rows, groups of 32 gate and
// 32 up rows in turn; C = silu(gate) * up).  A few rows stream the weights once, more rows take the tensor-core GEMM.
struct RowsOut {
  const float* bias = nullptr;   // [N], added to the sums
  float softcap = 0.f;           // EPI_F32: cap tanh(c / cap) when not 0
  // columns n2 and up (0: none) go elsewhere: column n of row m to C2 + (m / T2) * stride2 + (m % T2) * ld2 + n - n2
  int n2 = 0, T2 = 1;
  void* C2 = nullptr;
  long long ld2 = 0, stride2 = 0;
};
template <typename T>
int rows_linear(DecoderStack* d, const void* X, long long ldx, const void* W, long long ldw, void* C, long long ldc, int M, int N, int K,
                int epi, cudaStream_t s, const RowsOut& out = RowsOut());

// The streaming kernel by itself (bf16, aligned, at most ROWS_STREAM rows), as a batch over heads: element strides between the
// heads' operands, and optionally one gate logit per (row, head) whose sigmoid multiplies the result.
constexpr int ROWS_STREAM = 32;
struct RowsBatch {
  long long x = 0, w = 0, c = 0;
  const bf16* gate = nullptr;
  long long ld_gate = 0;
  RowsOut out;
  // Experts: the batch are the lists of k_moe_choose_few (lists[0] of them, each expert, start, length); list entry p is row
  // p / x_div of X and row p of C; EPI_RELU2 squares the positive part of the result.
  const int* lists = nullptr;
  int max_lists = 0, x_div = 1;
};
int rows_stream(const bf16* X, long long ldx, const bf16* W, long long ldw, void* C, long long ldc, int M, int N, int K, int epi, int batch,
                const RowsBatch& bt, cudaStream_t s);

// ---- recurrences (recurrence.cu) ------------------------------------------------------------------------------------
struct RecurrenceArgs {
  const void *q = nullptr, *k = nullptr, *v = nullptr;   // q, k: fp32 rows when qk_f32, else the compute type with silu applied here
  long long ldq = 0, ldk = 0, ldv = 0;
  const float* g = nullptr;      // [rows][heads * dim] decays per channel, or NULL: decay[heads]
  const float* beta = nullptr;   // [rows][heads], or NULL: plain sum of outer products
  const float* decay = nullptr;
  float* S = nullptr;            // [B][heads][vdim][dim]
  void* o = nullptr;             // [rows][heads * vdim]
  int B = 0, T = 0, heads = 0, qk_heads = 0, dim = 0, vdim = 0;
};
template <typename T> int recurrence(const RecurrenceArgs& a, cudaStream_t s);

// Short causal convolutions + silu, unit vectors, decays and step sizes of the gated delta rule.
struct DeltaPrepArgs {
  const void* proj = nullptr; long long ldp = 0;
  int s_q = 0, s_k = 0, s_v = 0, s_b = 0;
  const float *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr, *a_log = nullptr, *dt_bias = nullptr;
  const void* tail_in = nullptr; void* tail_out = nullptr;
  float *qn = nullptr, *kn = nullptr, *gd = nullptr, *beta = nullptr; void* vv = nullptr;   // gd holds W_a2 W_a1 h on entry
  int B = 0, T = 0, heads = 0, kv_heads = 0, dim = 0, vdim = 0, taps = 0;
};
template <typename T> int delta_prep(const DeltaPrepArgs& a, cudaStream_t s);
template <typename T> int conv_tail(const DeltaPrepArgs& a, cudaStream_t s);   // only the kept inputs

// One token per column: everything between the packed projection and the output projection in one launch.
struct DeltaDecodeArgs {
  DeltaPrepArgs p;               // projections, taps and kept inputs (its outputs are unused)
  int s_a1 = 0, s_g1 = 0, ra = 0, rg = 0;
  const void *w_a2 = nullptr, *w_g2 = nullptr;
  float* S = nullptr;
  const float* norm = nullptr; float eps = 0.f;
  void* out = nullptr;           // [B][heads * vdim], normed and gated
};
template <typename T> int delta_decode(const DeltaDecodeArgs& a, cudaStream_t s);

// The same recurrences for many tokens in bf16 models, chunk by chunk on the tensor cores (chunked_recurrence.cu);
// convolutions, unit vectors and decays included.
struct ChunkArgs {
  const void* proj = nullptr; long long ldp = 0;        // packed projections; q, k (and v, without convolutions) get silu here
  int s_q = 0, s_k = 0, s_v = 0, s_b = 0;
  const float *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr, *a_log = nullptr, *dt_bias = nullptr;
  const float* graw = nullptr;   // [rows][heads * dim] W_a2 W_a1 h, or NULL: decayed sum with decay[heads]
  const float* decay = nullptr;
  const void* tail_in = nullptr;
  float* S = nullptr; void* o = nullptr;
  int B = 0, T = 0, heads = 0, qk_heads = 0, dim = 0, vdim = 0, taps = 1;
  char* ws = nullptr; size_t ws_bytes = 0;
  unsigned int* status = nullptr;
  int t0 = 0, chunks = 0; size_t item_bytes = 0;        // set per segment
};
size_t chunked_recurrence_item_bytes(int dim, int vdim);
bool chunked_recurrence_supported(const ChunkArgs& a);
int chunked_recurrence(const ChunkArgs& a, cudaStream_t s);

// ---- latent attention (latent_attention.cu) -------------------------------------------------------------------------
struct LatentArgs {
  void* q = nullptr;             // [rows][heads (dim + rot_dim)], not rotated yet
  const void* dkv = nullptr; long long ld_dkv = 0;     // new rows of W_dkv h (kv_rank, rot_dim)
  const float* dkv_norm = nullptr;
  const void* gate = nullptr; long long ld_gate = 0;   // one logit per head
  void* latent = nullptr;        // cache [maxB][maxT][ld]
  int ld = 0, lp = 0, maxT = 0;
  const void* w_kv = nullptr;    // [heads dim + heads vdim][lp]
  const void* w_ukt = nullptr;   // [heads][lp][dp]: the key up-projection transposed, dim padded to dp
  int dp = 0;
  void* oc = nullptr;            // [rows][heads][lp] attention results in the latent space
  void* kv = nullptr;            // expanded keys and values, [B][maxT][heads (dim + vdim)]
  float* qabs = nullptr; float* part = nullptr; size_t part_floats = 0;
  void* o = nullptr;             // [rows][heads vdim]
  int B = 0, T = 0, first = 0, heads = 0, dim = 0, rot_dim = 0, rot_dims = 0, vdim = 0, kv_rank = 0;
  float scale = 1.f, eps = 0.f;
  const float* freq = nullptr;   // [rot_dims / 2] angle per position
  const void* dq = nullptr; const float* dq_norm = nullptr; void* cq = nullptr; int q_rank = 0, qp = 0;   // query latent
  DecoderStack* d = nullptr;
};
template <typename T> int latent_norms(const LatentArgs& a, cudaStream_t s);   // query latent -> cq, new rows -> cache
template <typename T> int latent_attention(const LatentArgs& a, cudaStream_t s);
bool latent_attention_tc_supported(const LatentArgs& a);       // slab_attention_sm100.cu: the prompt's attention on the tensor cores
int latent_attention_tc(const LatentArgs& a, cudaStream_t s);

// ---- attention over cached keys and values (window_attention.cu; prompts in bf16: slab_attention_sm100.cu) --------------
struct WindowAttnArgs {
  const void* q = nullptr; long long ldq = 0;          // [rows][heads][maps][dim]
  const void* kv = nullptr;      // cache [maxB][maxT][ld]: keys [kv_heads][maps][dim], from column vo on values [kv_heads][vdim]
  int ld = 0, vo = 0, maxT = 0;
  const void* gate = nullptr; long long ld_gate = 0; int gate_mode = FEMTO_GATE_NONE;   // [rows][heads] or [rows][heads vdim]
  void* o = nullptr;             // [rows][heads vdim]
  int B = 0, T = 0, first = 0, heads = 0, kv_heads = 0, dim = 0, vdim = 0, maps = 1, window = 0, keep = 0;
  float scale = 1.f, eps = 0.f, out_scale = 1.f;
  const float* sink = nullptr;   // [heads]
  const float* lambda = nullptr; // two maps: (a1 - lambda a2) / rms * out_scale
  float* part = nullptr; size_t part_floats = 0;
  unsigned int* status = nullptr;
};
template <typename T> int qk_norm(const WindowAttnArgs& a, const float* wq, const float* wk, bool with_k, cudaStream_t s);   // in place
template <typename T> int window_attention(const WindowAttnArgs& a, cudaStream_t s);
int diff_lambda(const float* lq1, const float* lk1, const float* lq2, const float* lk2, int dim, float diff, float* out, cudaStream_t s);
size_t window_attention_part_floats(int max_batch, int heads, int maps, int vdim);
bool window_attention_tc_supported(const WindowAttnArgs& a);
int window_attention_tc(const WindowAttnArgs& a, cudaStream_t s);
constexpr int ATTN_FEW = 8;            // columns with at most this many new tokens take the split-key kernels

// ---- mixture of experts (moe.cu) -------------------------------------------------------------------------------------
struct MoeArgs {
  const float* z = nullptr; long long ldz = 0;         // router logits [rows][ldz], without the bias
  const float* bias = nullptr;
  const void* router = nullptr;  // instead of z: router weights [experts][width], at most MOE_ROUTE of them in bf16
  int rows = 0, experts = 0, top = 0, width = 0, group_rows = 0, max_lists = 0;
  const void* h = nullptr;       // [rows][width]
  float* weight = nullptr; int *expert = nullptr, *slot = nullptr;   // [rows * top]
  int* counts = nullptr;         // [experts]
  int* groups = nullptr;         // runs of the sorted rows: their number, then the expert of each
  int* lists = nullptr;          // few rows: number of lists, (expert, start, length) of each, from 1 + 3 max_lists on the pairs
  void* xs = nullptr;            // sorted inputs
};
constexpr int MOE_ROUTE = 64;          // experts up to which moe_sort can multiply by the router itself
bool moe_supported(int experts, int top);
int moe_group_rows(long long rows, int experts, int top);
long long moe_max_slots(long long rows, int experts, int top, int group_rows);
template <typename T> int moe_sort(const MoeArgs& a, cudaStream_t s);
int moe_choose_few(const MoeArgs& a, cudaStream_t s);
template <typename T> int moe_combine(const MoeRows& m, T* y, int rows, int d, cudaStream_t s);

constexpr int LATENT_FEW = 8;          // columns with at most this many new tokens attend in the latent space
constexpr int LATENT_MAX_SPLITS = 64;

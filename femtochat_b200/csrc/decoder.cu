// Decoders given as a list of layers: configuration, flat layout, packed weights, cache and the forward schedule.  One
// schedule serves prompts, portions of prompts and single tokens: it runs the tokens it is given from the states that
// earlier calls left.
#include "decoder.cuh"

#include <math.h>
#include <string.h>

#include <algorithm>

#include "streaming.cuh"

// ---- configuration and layout -------------------------------------------------------------------------------------
static int check_layer(const femto_decoder_config& cfg, int i) {
  const femto_layer_config& c = cfg.h_layers[i];
#define NEED(cond, what) if (!(cond)) return femto_fail(FEMTO_ERR_SHAPE, "layer %d: %s", i, what)
  NEED(c.heads > 0 && c.dim > 0 && c.vdim > 0, "heads, dim and vdim must be positive");
  NEED(c.ff >= 0, "ff is negative");
  NEED(c.weights_of < cfg.n_layer && c.weights_of != i, "weights_of names no other layer");
  if (c.experts) NEED(c.ff > 0 && moe_supported(c.experts, c.top), "a mixture needs 1 to 1024 experts, of which a token uses 1 to 32, and their ff");
  switch (c.mixer) {
    case FEMTO_MIXER_LIGHTNING:
      NEED(c.h_decay != nullptr, "lightning attention needs one decay per head");
      NEED(c.dim <= 256, "dim above 256 is not supported");
      break;
    case FEMTO_MIXER_CHANNEL_DELTA:
      NEED(c.kv_heads > 0 && c.heads % c.kv_heads == 0, "heads must be a multiple of kv_heads");
      NEED(c.conv >= 1, "conv must be positive");
      NEED(c.decay_rank > 0 && c.gate_rank > 0, "the low-rank projections need a rank");
      NEED(c.dim <= 256 && c.vdim <= 256, "dim or vdim above 256 is not supported");
      break;
    case FEMTO_MIXER_LATENT_ATTENTION:
      NEED(c.q_rank > 0 && c.kv_rank > 0 && c.rot_dim >= 0, "q_rank and kv_rank must be positive");
      NEED(c.rot_dims >= 0 && c.rot_dims <= c.rot_dim && c.rot_dims % 2 == 0, "rot_dims must be even and at most rot_dim");
      NEED(c.kv_rank <= 1024 && c.vdim <= 256 && c.dim + c.rot_dim <= 512, "kv_rank above 1024, vdim above 256 or dim + rot_dim above 512 is not supported");
      break;
    case FEMTO_MIXER_ATTENTION:
      NEED(c.kv_heads > 0 && c.heads % c.kv_heads == 0, "heads must be a multiple of kv_heads");
      NEED(c.maps == 1 || c.maps == 2, "maps must be 1 or 2");
      NEED(c.window > 0 && c.keep_first >= 0, "window must be positive and keep_first not negative");
      NEED(c.gate >= FEMTO_GATE_NONE && c.gate <= FEMTO_GATE_ELEMENT, "unknown gate");
      NEED(c.dim <= 256 && c.vdim <= 256, "dim or vdim above 256 is not supported");
      if (c.kv_from >= 0) {
        NEED(c.kv_from < i, "kv_from must name an earlier layer");
        const femto_layer_config& o = cfg.h_layers[c.kv_from];
        NEED(o.mixer == FEMTO_MIXER_ATTENTION && o.kv_from < 0, "kv_from must name an attention layer with keys and values of its own");
        NEED(o.kv_heads == c.kv_heads && o.dim == c.dim && o.vdim == c.vdim && o.maps == c.maps, "differs in its key or value sizes from the layer named by kv_from");
      }
      break;
    default: return femto_fail(FEMTO_ERR_ARG, "layer %d: unknown mixer %d", i, c.mixer);
  }
#undef NEED
  return 0;
}

int decoder_fill(DecoderStack* d, const femto_decoder_config* cfg) {
  if (!cfg || !cfg->h_layers) return femto_fail(FEMTO_ERR_ARG, "config is NULL");
  if (cfg->vocab <= 0 || cfg->width <= 0 || cfg->n_layer <= 0) return femto_fail(FEMTO_ERR_ARG, "vocab, width and n_layer must be positive");
  if (cfg->compute_dtype != FEMTO_F32 && cfg->compute_dtype != FEMTO_BF16) return femto_fail(FEMTO_ERR_ARG, "compute_dtype must be FEMTO_F32 or FEMTO_BF16");
  if (cfg->index_base != 0 && cfg->index_base != 1) return femto_fail(FEMTO_ERR_ARG, "index_base must be 0 or 1");
  if (cfg->block != FEMTO_BLOCK_SANDWICH && cfg->block != FEMTO_BLOCK_PARALLEL) return femto_fail(FEMTO_ERR_ARG, "unknown block %d", cfg->block);
  d->cfg = *cfg;
  d->layer_cfg.assign(cfg->h_layers, cfg->h_layers + cfg->n_layer);
  d->cfg.h_layers = d->layer_cfg.data();
  d->bf = cfg->compute_dtype == FEMTO_BF16;
  d->layers.assign(cfg->n_layer, DecLayer());
  for (int i = 0; i < cfg->n_layer; i++) {
    FEMTO_TRY(check_layer(*cfg, i));
    DecLayer& l = d->layers[i];
    l.c = cfg->h_layers[i];
    l.own = i;
    for (int hops = 0; d->layer_cfg[l.own].weights_of >= 0; hops++) {
      if (hops > cfg->n_layer) return femto_fail(FEMTO_ERR_SHAPE, "layer %d: weights_of goes round in a circle", i);
      l.own = d->layer_cfg[l.own].weights_of;
    }
    const femto_layer_config &a = l.c, &o = d->layer_cfg[l.own];
    if (a.mixer != o.mixer || a.heads != o.heads || a.kv_heads != o.kv_heads || a.dim != o.dim || a.vdim != o.vdim || a.conv != o.conv ||
        a.q_rank != o.q_rank || a.kv_rank != o.kv_rank || a.rot_dim != o.rot_dim || a.ff != o.ff || a.maps != o.maps || a.qkv_bias != o.qkv_bias ||
        a.qk_norm != o.qk_norm || a.sink != o.sink || a.gate != o.gate || (a.kv_from < 0) != (o.kv_from < 0) || a.diff != o.diff || a.experts != o.experts)
      return femto_fail(FEMTO_ERR_SHAPE, "layer %d differs in its sizes from layer %d, whose weights it uses", i, l.own);
    l.c.decay_rank = o.decay_rank; l.c.gate_rank = o.gate_rank;
    if (a.mixer == FEMTO_MIXER_LIGHTNING) l.decay.assign(a.h_decay, a.h_decay + a.heads);
    l.c.h_decay = nullptr;
    if (a.mixer == FEMTO_MIXER_LATENT_ATTENTION)
      for (int k = 0; k < a.rot_dims / 2; k++) l.freq.push_back((float)pow(a.rot_base, -2.0 * k / a.rot_dims));
  }
  // flat layout, and the derived sizes of every layer
  long long pos = 0;
  d->tensors.clear();
  auto take = [&](const std::string& name, long long rows, long long cols) {
    femto_decoder_tensor t;
    memset(&t, 0, sizeof(t));
    strncpy(t.name, name.c_str(), sizeof(t.name) - 1);
    t.offset = pos; t.rows = rows; t.cols = cols;
    pos += (rows * std::max(1LL, cols) + 3) / 4 * 4;   // every tensor on a 16-byte boundary
    d->tensors.push_back(t);
    return t.offset;
  };
  const long long w = cfg->width;
  const bool sandwich = cfg->block == FEMTO_BLOCK_SANDWICH;
  d->off_embed = take("embed", cfg->vocab, w);
  for (int i = 0; i < cfg->n_layer; i++) {
    DecLayer& l = d->layers[i];
    const femto_layer_config& c = l.c;
    const long long H = c.heads, D = c.dim, E = c.vdim, G = c.kv_heads;
    auto seg = [&](long long n) { const int at = l.n_in; l.n_in += round_up((int)n, 8); return at; };
    l.ffp = round_up(c.ff, c.experts ? 8 : 32);
    const std::string p = "l" + std::to_string(i) + ".", x = p + "mix.";
    const bool mine = l.own == i;
    auto put = [&](const std::string& name, long long rows, long long cols) { return mine ? take(name, rows, cols) : -1LL; };
    l.norm1 = put(p + "norm1", w, 0);
    if (sandwich) l.norm1b = put(p + "norm1b", w, 0);
    if (c.mixer == FEMTO_MIXER_LIGHTNING) {
      l.s_q = seg(H * D); l.s_k = seg(H * D); l.s_v = seg(H * E); l.s_g = seg(H * E);
      put(x + "q", H * D, w); put(x + "k", H * D, w); put(x + "v", H * E, w); put(x + "g", H * E, w);
      l.mix_norm = put(x + "norm", H * E, 0);
    } else if (c.mixer == FEMTO_MIXER_CHANNEL_DELTA) {
      l.ra = round_up(c.decay_rank, 8); l.rg = round_up(c.gate_rank, 8);
      l.s_q = seg(G * D); l.s_k = seg(G * D); l.s_v = seg(H * E); l.s_b = seg(H); l.s_a1 = seg(c.decay_rank); l.s_g1 = seg(c.gate_rank);
      put(x + "q", G * D, w); put(x + "k", G * D, w); put(x + "v", H * E, w); put(x + "b", H, w);
      put(x + "a1", c.decay_rank, w); put(x + "g1", c.gate_rank, w);
      put(x + "a2", H * D, c.decay_rank); put(x + "g2", H * E, c.gate_rank);
      l.conv_q = put(x + "q.conv", G * D, c.conv); l.conv_k = put(x + "k.conv", G * D, c.conv); l.conv_v = put(x + "v.conv", H * E, c.conv);
      l.a_log = put(x + "A_log", H, 0); l.dt_bias = put(x + "dt_bias", H * D, 0); l.mix_norm = put(x + "norm", E, 0);
    } else if (c.mixer == FEMTO_MIXER_ATTENTION) {
      // q and the gate are columns of proj; keys and values go from the same product straight to the cache
      const long long M = c.maps;
      const bool own_kv = c.kv_from < 0;
      l.s_q = seg(H * M * D);
      if (c.gate != FEMTO_GATE_NONE) l.s_g = seg(c.gate == FEMTO_GATE_HEAD ? H : H * E);
      l.vo = round_up((int)(G * M * D), 8);
      l.n_kv = l.vo + round_up((int)(G * E), 8);
      l.kv_layer = own_kv ? i : c.kv_from;
      put(x + "q", H * M * D, w);
      if (own_kv) { put(x + "k", G * M * D, w); put(x + "v", G * E, w); }
      if (c.qkv_bias) {
        l.q_bias = put(x + "q.b", H * M * D, 0);
        if (own_kv) { l.k_bias = put(x + "k.b", G * M * D, 0); l.v_bias = put(x + "v.b", G * E, 0); }
      }
      if (c.qk_norm) { l.q_norm = put(x + "q.norm", D, 0); if (own_kv) l.k_norm = put(x + "k.norm", D, 0); }
      if (M == 2) { l.lq1 = put(x + "lq1", D, 0); l.lk1 = put(x + "lk1", D, 0); l.lq2 = put(x + "lq2", D, 0); l.lk2 = put(x + "lk2", D, 0); }
      if (c.sink) l.sink = put(x + "sink", H, 0);
      if (c.gate != FEMTO_GATE_NONE) put(x + "g", c.gate == FEMTO_GATE_HEAD ? H : H * E, w);
    } else {
      l.qp = round_up(c.q_rank, 8); l.dp = round_up(c.dim, 8); l.lp = round_up(c.kv_rank, 8); l.ld = round_up(l.lp + c.rot_dim, 8);
      l.s_q = seg(c.q_rank); l.s_dkv = seg(c.kv_rank + c.rot_dim); l.s_g = seg(H);
      put(x + "dq", c.q_rank, w); put(x + "dkv", c.kv_rank + c.rot_dim, w); put(x + "g", H, w);
      put(x + "uq", H * (D + c.rot_dim), c.q_rank); put(x + "uk", H * D, c.kv_rank); put(x + "uv", H * E, c.kv_rank);
      l.dq_norm = put(x + "dq.norm", c.q_rank, 0); l.dkv_norm = put(x + "dkv.norm", c.kv_rank, 0);
    }
    put(x + "o", w, H * E);
    if (c.ff > 0) {
      l.norm2 = put(p + "norm2", w, 0);
      if (sandwich) l.norm2b = put(p + "norm2b", w, 0);
      if (c.experts) {
        put(p + "mlp.router", c.experts, w);
        l.router_bias = put(p + "mlp.router.b", c.experts, 0);
        for (int e = 0; e < c.experts; e++) {
          const std::string x2 = p + "mlp.e" + std::to_string(e);
          put(x2 + ".up", c.ff, w); put(x2 + ".down", w, c.ff);
        }
      } else {
        put(p + "mlp.gate", c.ff, w); put(p + "mlp.up", c.ff, w); put(p + "mlp.down", w, c.ff);
      }
    }
  }
  for (auto& l : d->layers) {
    const DecLayer& o = d->layers[l.own];
    l.norm1 = o.norm1; l.norm1b = o.norm1b; l.norm2 = o.norm2; l.norm2b = o.norm2b; l.mix_norm = o.mix_norm; l.conv_q = o.conv_q;
    l.conv_k = o.conv_k; l.conv_v = o.conv_v; l.a_log = o.a_log; l.dt_bias = o.dt_bias; l.dq_norm = o.dq_norm; l.dkv_norm = o.dkv_norm;
    l.q_norm = o.q_norm; l.k_norm = o.k_norm; l.sink = o.sink; l.q_bias = o.q_bias; l.k_bias = o.k_bias; l.v_bias = o.v_bias;
    l.lq1 = o.lq1; l.lk1 = o.lk1; l.lq2 = o.lq2; l.lk2 = o.lk2; l.router_bias = o.router_bias;
  }
  if (cfg->untied) take("head", cfg->vocab, w);
  d->off_final = take("final.norm", w, 0);
  d->nparams = pos;
  return 0;
}

// ---- weights and workspace ------------------------------------------------------------------------------------------
namespace {
struct Carver {
  char* base = nullptr;
  size_t off = 0;
  template <typename P> void take(P*& p, size_t bytes) {
    off = (off + 255) & ~(size_t)255;
    p = base ? reinterpret_cast<P*>(base + off) : nullptr;
    off += bytes;
  }
};

void carve(DecoderStack* d, Carver& b) {
  const size_t es = d->bf ? 2 : 4, R = d->cfg.max_rows, w = d->cfg.width;
  b.take(d->status, 256);
  b.take(d->embed, es * d->cfg.vocab * w);
  d->head = d->embed;
  if (d->cfg.untied) b.take(d->head, es * d->cfg.vocab * w);
  size_t moe_pairs = 0, experts = 0, slots_w = 0, slots_ff = 0, runs = 0;
  bool dense = false;
  size_t n_in = 0, mix = 0, ff = 0, qk = 0, hd = 0, heads = 0, g2 = 0, cq = 0, q = 0, qa = 0, vv = 0;
  for (size_t i = 0; i < d->layers.size(); i++) {
    DecLayer& l = d->layers[i];
    const femto_layer_config& c = l.c;
    const size_t H = c.heads, D = c.dim, E = c.vdim;
    n_in = std::max(n_in, (size_t)l.n_in); mix = std::max(mix, H * E); ff = std::max(ff, (size_t)l.ffp);
    if (c.mixer == FEMTO_MIXER_CHANNEL_DELTA) {
      qk = std::max(qk, c.kv_heads * D); hd = std::max(hd, H * D); heads = std::max(heads, H); g2 = std::max(g2, H * E); vv = std::max(vv, H * E);
    }
    if (c.mixer == FEMTO_MIXER_LATENT_ATTENTION) {
      cq = std::max(cq, (size_t)l.qp); q = std::max(q, H * (D + c.rot_dim)); qa = std::max(qa, H * l.ld);
    }
    if (c.ff > 0 && !c.experts) dense = true;
    if (c.experts) {
      for (const int gr : {128, 256}) {
        const size_t slots = moe_max_slots(R, c.experts, c.top, gr);
        slots_w = std::max(slots_w, slots); slots_ff = std::max(slots_ff, slots * l.ffp); runs = std::max(runs, slots / gr);
      }
      moe_pairs = std::max(moe_pairs, R * c.top); experts = std::max(experts, (size_t)c.experts);
    }
    b.take(l.decay_dev, 4 * H);
    b.take(l.freq_dev, 4 * l.freq.size() + 4);
    if (l.own != (int)i) continue;
    const bool own_kv = c.mixer == FEMTO_MIXER_ATTENTION && c.kv_from < 0;
    b.take(l.w_in, es * (l.n_in + (own_kv ? l.n_kv : 0)) * w); b.take(l.w_o, es * w * H * E);
    if (c.mixer == FEMTO_MIXER_ATTENTION) {
      if (c.qkv_bias) b.take(l.bias, 4 * (size_t)(l.n_in + l.n_kv));
      b.take(l.lambda, 4);
    }
    if (c.mixer == FEMTO_MIXER_CHANNEL_DELTA) { b.take(l.w_a2, es * H * D * l.ra); b.take(l.w_g2, es * H * E * l.rg); }
    if (c.mixer == FEMTO_MIXER_LATENT_ATTENTION) { b.take(l.w_uq, es * H * (D + c.rot_dim) * l.qp); b.take(l.w_kv, es * H * (D + E) * l.lp); b.take(l.w_ukt, es * H * l.lp * l.dp); }
    if (c.experts) {
      b.take(l.w_router, es * c.experts * w); b.take(l.w_gu, es * c.experts * l.ffp * w); b.take(l.w_down, es * c.experts * w * l.ffp);
    } else if (c.ff > 0) { b.take(l.w_gu, es * 2 * l.ffp * w); b.take(l.w_down, es * w * l.ffp); }
  }
  for (auto& l : d->layers) {
    const DecLayer& o = d->layers[l.own];
    l.w_in = o.w_in; l.w_o = o.w_o; l.w_a2 = o.w_a2; l.w_g2 = o.w_g2; l.w_uq = o.w_uq; l.w_kv = o.w_kv; l.w_ukt = o.w_ukt; l.w_gu = o.w_gu; l.w_down = o.w_down;
    l.w_router = o.w_router; l.bias = o.bias; l.lambda = o.lambda;
  }
  b.take(d->tok0, 4 * R); b.take(d->want, 4 * R);
  b.take(d->x, 4 * R * w); b.take(d->hn, es * R * w); b.take(d->y, es * R * w);
  if (d->cfg.block == FEMTO_BLOCK_PARALLEL) { b.take(d->hn2, es * R * w); if (dense) b.take(d->y2, es * R * w); }
  b.take(d->moe_z, 4 * R * round_up((int)experts, 4)); b.take(d->moe_weight, 4 * moe_pairs); b.take(d->moe_expert, 4 * moe_pairs);
  b.take(d->moe_slot, 4 * moe_pairs); b.take(d->moe_counts, 4 * experts); b.take(d->moe_groups, 4 * (runs + 1));
  const size_t few_pairs = experts ? (size_t)ROWS_STREAM * 32 : 0;
  b.take(d->moe_lists, 4 * (1 + 4 * few_pairs));
  b.take(d->moe_x, es * slots_w * w); b.take(d->moe_act, es * slots_ff); b.take(d->moe_out, es * slots_w * w);
  b.take(d->proj, es * R * n_in); b.take(d->mixo, es * R * mix); b.take(d->mixg, es * R * mix);
  b.take(d->gu, es * R * 2 * ff); b.take(d->act, es * R * ff);
  b.take(d->qn, 4 * R * qk); b.take(d->kn, 4 * R * qk); b.take(d->gd, 4 * R * hd); b.take(d->beta, 4 * R * heads);
  b.take(d->vv, es * R * vv); b.take(d->g2, es * R * g2);
  b.take(d->cq, es * R * cq); b.take(d->q, es * R * q);
  const size_t few = std::min(R, (size_t)d->cfg.max_batch * LATENT_FEW);
  b.take(d->qabs, 4 * few * qa); b.take(d->oc, es * few * qa);
  size_t items = 0;
  for (const auto& l : d->layers)
    if (d->bf && l.c.mixer != FEMTO_MIXER_LATENT_ATTENTION && l.c.dim <= 128 && l.c.vdim <= 128)
      items = std::max(items, chunked_recurrence_item_bytes(l.c.dim, l.c.vdim) * l.c.heads * d->cfg.max_batch);
  // operands of the chunks of one segment, at least one chunk of every column
  const size_t chunks = items ? std::max<size_t>(1, std::min<size_t>(((size_t)160 << 20) / items, R / d->cfg.max_batch / 64 + 1)) : 0;
  d->chunk_ws_bytes = items * chunks;
  b.take(d->chunk_ws, d->chunk_ws_bytes);
  d->gemm_ws_bytes = (size_t)64 << 20;
  b.take(d->gemm_ws, d->gemm_ws_bytes);
}
}  // namespace

int decoder_create(const femto_decoder_config* cfg, femto_handle** out) {
  DecoderStack* d = new DecoderStack();
  int r = decoder_fill(d, cfg);
  if (!r && (cfg->max_batch <= 0 || cfg->max_rows < cfg->max_batch)) r = femto_fail(FEMTO_ERR_ARG, "max_batch must be positive and max_rows at least max_batch");
  if (r) { delete d; return r; }
  Carver dry;
  carve(d, dry);
  const size_t bytes = dry.off + 256;
  cudaError_t e = cudaMalloc(&d->arena, bytes);
  if (e == cudaSuccess) e = cudaMemset(d->arena, 0, bytes);   // padding columns of packed weights stay zero
  if (e != cudaSuccess) {
    r = femto_fail(FEMTO_ERR_NOMEM, "%.2f GiB of weights and workspace: %s", bytes / 1073741824.0, cudaGetErrorString(e));
    if (d->arena) cudaFree(d->arena);
    delete d;
    return r;
  }
  Carver real;
  real.base = d->arena;
  carve(d, real);
  for (auto& l : d->layers) {
    if (!l.freq.empty()) cudaMemcpy(l.freq_dev, l.freq.data(), 4 * l.freq.size(), cudaMemcpyHostToDevice);
    if (!l.decay.empty()) cudaMemcpy(l.decay_dev, l.decay.data(), 4 * l.decay.size(), cudaMemcpyHostToDevice);
  }
  femto_handle* h = new femto_handle();
  h->dec = d;
  h->bf = d->bf;
  h->nparams = d->nparams;
  h->maxB = cfg->max_batch;
  h->status = d->status;
  e = cudaDeviceSynchronize();
  if (e != cudaSuccess) { r = femto_fail((int)e, "device error while creating the decoder: %s", cudaGetErrorString(e)); decoder_free(d); delete h; return r; }
  *out = h;
  return 0;
}

void decoder_free(DecoderStack* d) {
  if (!d) return;
  if (d->arena) cudaFree(d->arena);
  delete d;
}

template <typename T> static int refresh_t(DecoderStack* d, const float* theta, cudaStream_t s) {
  auto find = [&](const std::string& name) -> const femto_decoder_tensor* {
    for (const auto& t : d->tensors) if (name == t.name) return &t;
    return nullptr;
  };
  const int w = d->cfg.width;
  auto pack = [&](const std::string& name, void* dst, int ldd, int row, int group, int step) {
    const femto_decoder_tensor* t = find(name);
    if (!t) return femto_fail(FEMTO_ERR_STATE, "no tensor %s", name.c_str());
    return pack_rows<T>(theta + t->offset, (int)t->rows, (int)t->cols, (T*)dst, ldd, row, group, step, s);
  };
  const int all = 1 << 30;
  FEMTO_TRY(pack("embed", d->embed, w, 0, all, 0));
  if (d->cfg.untied) FEMTO_TRY(pack("head", d->head, w, 0, all, 0));
  for (size_t i = 0; i < d->layers.size(); i++) {
    DecLayer& l = d->layers[i];
    if (l.own != (int)i) continue;
    const femto_layer_config& c = l.c;
    const std::string p = "l" + std::to_string(i) + ".", x = p + "mix.";
    if (c.mixer == FEMTO_MIXER_ATTENTION) {
      FEMTO_TRY(pack(x + "q", l.w_in, w, l.s_q, all, 0));
      if (c.gate != FEMTO_GATE_NONE) FEMTO_TRY(pack(x + "g", l.w_in, w, l.s_g, all, 0));
      if (c.kv_from < 0) { FEMTO_TRY(pack(x + "k", l.w_in, w, l.n_in, all, 0)); FEMTO_TRY(pack(x + "v", l.w_in, w, l.n_in + l.vo, all, 0)); }
      if (c.qkv_bias) {
        auto put_bias = [&](long long off, int at, int n) {
          return cudaMemcpyAsync(l.bias + at, theta + off, 4 * (size_t)n, cudaMemcpyDeviceToDevice, s);
        };
        CUDA_TRY(put_bias(l.q_bias, l.s_q, c.heads * c.maps * c.dim));
        if (c.kv_from < 0) { CUDA_TRY(put_bias(l.k_bias, l.n_in, c.kv_heads * c.maps * c.dim)); CUDA_TRY(put_bias(l.v_bias, l.n_in + l.vo, c.kv_heads * c.vdim)); }
      }
      if (c.maps == 2) FEMTO_TRY(diff_lambda(theta + l.lq1, theta + l.lk1, theta + l.lq2, theta + l.lk2, c.dim, c.diff, l.lambda, s));
    } else if (c.mixer == FEMTO_MIXER_LATENT_ATTENTION) {
      FEMTO_TRY(pack(x + "dq", l.w_in, w, l.s_q, all, 0)); FEMTO_TRY(pack(x + "dkv", l.w_in, w, l.s_dkv, all, 0));
      FEMTO_TRY(pack(x + "g", l.w_in, w, l.s_g, all, 0));
      FEMTO_TRY(pack(x + "uq", l.w_uq, l.qp, 0, all, 0));
      FEMTO_TRY(pack_transposed<T>(theta + find(x + "uk")->offset, c.heads, c.dim, c.kv_rank, (T*)l.w_ukt, l.dp, l.lp, s));
      FEMTO_TRY(pack(x + "uk", l.w_kv, l.lp, 0, all, 0)); FEMTO_TRY(pack(x + "uv", l.w_kv, l.lp, c.heads * c.dim, all, 0));
    } else {
      FEMTO_TRY(pack(x + "q", l.w_in, w, l.s_q, all, 0)); FEMTO_TRY(pack(x + "k", l.w_in, w, l.s_k, all, 0));
      FEMTO_TRY(pack(x + "v", l.w_in, w, l.s_v, all, 0));
      if (c.mixer == FEMTO_MIXER_LIGHTNING) {
        FEMTO_TRY(pack(x + "g", l.w_in, w, l.s_g, all, 0));
      } else {
        FEMTO_TRY(pack(x + "b", l.w_in, w, l.s_b, all, 0)); FEMTO_TRY(pack(x + "a1", l.w_in, w, l.s_a1, all, 0));
        FEMTO_TRY(pack(x + "g1", l.w_in, w, l.s_g1, all, 0));
        FEMTO_TRY(pack(x + "a2", l.w_a2, l.ra, 0, all, 0)); FEMTO_TRY(pack(x + "g2", l.w_g2, l.rg, 0, all, 0));
      }
    }
    FEMTO_TRY(pack(x + "o", l.w_o, c.heads * c.vdim, 0, all, 0));
    if (c.experts) {
      FEMTO_TRY(pack(p + "mlp.router", l.w_router, w, 0, all, 0));
      for (int e = 0; e < c.experts; e++) {
        const std::string x2 = p + "mlp.e" + std::to_string(e);
        FEMTO_TRY(pack(x2 + ".up", l.w_gu, w, e * l.ffp, all, 0)); FEMTO_TRY(pack(x2 + ".down", l.w_down, l.ffp, e * w, all, 0));
      }
    } else if (c.ff > 0) {   // groups of 32 gate rows and 32 up rows alternate, so that one epilogue sees both of a column
      FEMTO_TRY(pack(p + "mlp.gate", l.w_gu, w, 0, 32, 64)); FEMTO_TRY(pack(p + "mlp.up", l.w_gu, w, 32, 32, 64));
      FEMTO_TRY(pack(p + "mlp.down", l.w_down, l.ffp, 0, all, 0));
    }
  }
  d->weights_valid = true;
  return 0;
}

int decoder_refresh(femto_handle* h, const float* theta, cudaStream_t s) {
  return h->dec->bf ? refresh_t<bf16>(h->dec, theta, s) : refresh_t<float>(h->dec, theta, s);
}

// ---- cache ----------------------------------------------------------------------------------------------------------
int decoder_cache_create(femto_handle* h, int max_batch, int max_len, femto_kv_cache** out) {
  DecoderStack* d = h->dec;
  femto_kv_cache* c = new femto_kv_cache();
  c->h = h; c->maxB = max_batch; c->maxT = max_len;
  c->state.resize(d->layers.size());
  const size_t es = d->bf ? 2 : 4, B = max_batch;
  size_t exp_bytes = 0;
  for (auto& l : d->layers) {
    const femto_layer_config& q = l.c;
    if (q.mixer == FEMTO_MIXER_ATTENTION) c->part_floats = std::max(c->part_floats, window_attention_part_floats(max_batch, q.heads, q.maps, q.vdim));
    if (q.mixer != FEMTO_MIXER_LATENT_ATTENTION) continue;
    exp_bytes = std::max(exp_bytes, es * B * max_len * (size_t)q.heads * (q.dim + q.vdim));
    c->part_floats = std::max(c->part_floats, (size_t)std::max(128, max_batch * LATENT_FEW) * q.heads * (size_t)(l.lp + 2) * 2);
  }
  auto lay = [&](Carver& b) {
    for (size_t i = 0; i < d->layers.size(); i++) {
      const DecLayer& l = d->layers[i];
      const femto_layer_config& q = l.c;
      LayerState& s = c->state[i];
      if (q.mixer == FEMTO_MIXER_ATTENTION) {
        s.ld = l.n_kv;
        if (q.kv_from < 0) b.take(s.kv, es * B * max_len * l.n_kv);
      } else if (q.mixer != FEMTO_MIXER_LATENT_ATTENTION) { s.S_bytes = 4 * B * q.heads * q.dim * q.vdim; b.take(s.S, s.S_bytes); }
      if (q.mixer == FEMTO_MIXER_CHANNEL_DELTA) {
        s.tail_bytes = es * B * (q.conv - 1) * (2 * (size_t)q.kv_heads * q.dim + (size_t)q.heads * q.vdim);
        b.take(s.tail[0], s.tail_bytes); b.take(s.tail[1], s.tail_bytes);
      }
      if (q.mixer == FEMTO_MIXER_LATENT_ATTENTION) { s.ld = l.ld; b.take(s.latent, es * B * max_len * l.ld); }
    }
    b.take(c->part, 4 * c->part_floats);
    b.take(c->kv_exp, exp_bytes);
  };
  Carver dry;
  lay(dry);
  const size_t bytes = dry.off + 256;
  cudaError_t e = cudaMalloc(&c->mem, bytes);
  if (e == cudaSuccess) e = cudaMemset(c->mem, 0, bytes);
  if (e == cudaSuccess) e = cudaDeviceSynchronize();
  if (e != cudaSuccess) {
    if (c->mem) cudaFree(c->mem);
    delete c;
    return femto_fail(FEMTO_ERR_NOMEM, "%.2f GiB of cache: %s", bytes / 1073741824.0, cudaGetErrorString(e));
  }
  Carver real;
  real.base = c->mem;
  lay(real);
  *out = c;
  return 0;
}

int decoder_cache_reset(femto_kv_cache* c, cudaStream_t s) {
  for (auto& l : c->state) {
    if (l.S_bytes) FEMTO_TRY(fill_zero(l.S, l.S_bytes, s));
    if (l.tail_bytes) FEMTO_TRY(fill_zero(l.tail[l.tail_now], l.tail_bytes, s));
  }
  c->B = 0; c->len = 0;
  return 0;
}

// ---- forward ---------------------------------------------------------------------------------------------------------
template <typename T>
static int mixer_t(DecoderStack* d, femto_kv_cache* c, int i, const float* theta, int B, int Tn, int first, cudaStream_t s) {
  typedef DecStream<T> S;
  const DecLayer& l = d->layers[i];
  const femto_layer_config& q = l.c;
  LayerState& st = c->state[i];
  const int R = B * Tn, w = d->cfg.width, H = q.heads, D = q.dim, E = q.vdim;
  const float eps = d->cfg.norm_eps;
  T* proj = (T*)d->proj;
  T* out = (T*)d->mixg;
  if (q.mixer == FEMTO_MIXER_ATTENTION) {
    const LayerState& src = c->state[l.kv_layer];
    const bool own_kv = l.kv_layer == i;
    RowsOut ro;
    ro.bias = l.bias;
    if (own_kv) { ro.n2 = l.n_in; ro.T2 = Tn; ro.C2 = (T*)src.kv + (long long)first * src.ld; ro.ld2 = src.ld; ro.stride2 = (long long)c->maxT * src.ld; }
    FEMTO_TRY(rows_linear<T>(d, d->hn, w, l.w_in, w, proj, l.n_in, R, l.n_in + (own_kv ? l.n_kv : 0), w, EPI_STORE, s, ro));
    WindowAttnArgs a;
    a.q = proj + l.s_q; a.ldq = l.n_in; a.kv = src.kv; a.ld = src.ld; a.vo = l.vo; a.maxT = c->maxT;
    a.gate = proj + l.s_g; a.ld_gate = l.n_in; a.gate_mode = q.gate; a.o = out;
    a.B = B; a.T = Tn; a.first = first; a.heads = H; a.kv_heads = q.kv_heads; a.dim = D; a.vdim = E; a.maps = q.maps; a.window = q.window; a.keep = q.keep_first;
    a.scale = q.scale; a.eps = eps; a.out_scale = 1.f - q.diff; a.sink = q.sink ? theta + l.sink : nullptr; a.lambda = l.lambda;
    a.part = c->part; a.part_floats = c->part_floats; a.status = d->status;
    if (q.qk_norm) FEMTO_TRY(qk_norm<T>(a, theta + l.q_norm, own_kv ? theta + l.k_norm : nullptr, own_kv, s));
    FEMTO_TRY(window_attention<T>(a, s));
    return rows_linear<T>(d, out, H * E, l.w_o, H * E, d->y, w, R, w, H * E, EPI_STORE, s);
  }
  FEMTO_TRY(rows_linear<T>(d, d->hn, w, l.w_in, w, proj, l.n_in, R, l.n_in, w, EPI_STORE, s));
  if (q.mixer == FEMTO_MIXER_LIGHTNING) {
    ChunkArgs ca;
    ca.proj = proj; ca.ldp = l.n_in; ca.s_q = l.s_q; ca.s_k = l.s_k; ca.s_v = l.s_v; ca.decay = l.decay_dev; ca.S = st.S; ca.o = d->mixo;
    ca.B = B; ca.T = Tn; ca.heads = ca.qk_heads = H; ca.dim = D; ca.vdim = E; ca.ws = d->chunk_ws; ca.ws_bytes = d->chunk_ws_bytes; ca.status = d->status;
    RecurrenceArgs a;
    a.q = proj + l.s_q; a.k = proj + l.s_k; a.v = proj + l.s_v; a.ldq = a.ldk = a.ldv = l.n_in;
    a.decay = l.decay_dev; a.S = st.S; a.o = d->mixo; a.B = B; a.T = Tn; a.heads = a.qk_heads = H; a.dim = D; a.vdim = E;
    if (sizeof(T) == 2 && chunked_recurrence_supported(ca)) FEMTO_TRY(chunked_recurrence(ca, s));
    else FEMTO_TRY(recurrence<T>(a, s));
    FEMTO_TRY(S::gated_norm((const T*)d->mixo, theta + l.mix_norm, true, proj + l.s_g, l.n_in, out, R, 1, H * E, eps, s));
  } else if (q.mixer == FEMTO_MIXER_CHANNEL_DELTA) {
    DeltaPrepArgs p;
    p.proj = proj; p.ldp = l.n_in; p.s_q = l.s_q; p.s_k = l.s_k; p.s_v = l.s_v; p.s_b = l.s_b;
    p.conv_q = theta + l.conv_q; p.conv_k = theta + l.conv_k; p.conv_v = theta + l.conv_v; p.a_log = theta + l.a_log; p.dt_bias = theta + l.dt_bias;
    p.tail_in = st.tail[st.tail_now]; p.tail_out = st.tail[st.tail_now ^ 1];
    p.qn = d->qn; p.kn = d->kn; p.gd = d->gd; p.beta = d->beta; p.vv = d->vv;
    p.B = B; p.T = Tn; p.heads = H; p.kv_heads = q.kv_heads; p.dim = D; p.vdim = E; p.taps = q.conv;
    if (Tn == 1) {
      DeltaDecodeArgs t;
      t.p = p; t.s_a1 = l.s_a1; t.s_g1 = l.s_g1; t.ra = l.ra; t.rg = l.rg; t.w_a2 = l.w_a2; t.w_g2 = l.w_g2; t.S = st.S;
      t.norm = theta + l.mix_norm; t.eps = eps; t.out = out;
      FEMTO_TRY(delta_decode<T>(t, s));
      st.tail_now ^= 1;
      return rows_linear<T>(d, out, H * E, l.w_o, H * E, d->y, w, R, w, H * E, EPI_STORE, s);
    }
    FEMTO_TRY(rows_linear<T>(d, proj + l.s_a1, l.n_in, l.w_a2, l.ra, d->gd, H * D, R, H * D, l.ra, EPI_F32, s));
    FEMTO_TRY(rows_linear<T>(d, proj + l.s_g1, l.n_in, l.w_g2, l.rg, d->g2, H * E, R, H * E, l.rg, EPI_STORE, s));
    ChunkArgs ca;
    ca.proj = proj; ca.ldp = l.n_in; ca.s_q = l.s_q; ca.s_k = l.s_k; ca.s_v = l.s_v; ca.s_b = l.s_b; ca.conv_q = p.conv_q; ca.conv_k = p.conv_k;
    ca.conv_v = p.conv_v; ca.a_log = p.a_log; ca.dt_bias = p.dt_bias; ca.graw = d->gd; ca.tail_in = p.tail_in; ca.S = st.S; ca.o = d->mixo;
    ca.B = B; ca.T = Tn; ca.heads = H; ca.qk_heads = q.kv_heads; ca.dim = D; ca.vdim = E; ca.taps = q.conv; ca.ws = d->chunk_ws;
    ca.ws_bytes = d->chunk_ws_bytes; ca.status = d->status;
    const bool chunked = sizeof(T) == 2 && chunked_recurrence_supported(ca);
    if (chunked) { FEMTO_TRY(chunked_recurrence(ca, s)); FEMTO_TRY(conv_tail<T>(p, s)); }
    else FEMTO_TRY(delta_prep<T>(p, s));
    st.tail_now ^= 1;
    RecurrenceArgs a;
    a.q = d->qn; a.k = d->kn; a.v = d->vv; a.ldq = a.ldk = (long long)q.kv_heads * D; a.ldv = (long long)H * E;
    a.g = d->gd; a.beta = d->beta; a.S = st.S; a.o = d->mixo; a.B = B; a.T = Tn; a.heads = H; a.qk_heads = q.kv_heads; a.dim = D; a.vdim = E;
    if (!chunked) FEMTO_TRY(recurrence<T>(a, s));
    FEMTO_TRY(S::gated_norm((const T*)d->mixo, theta + l.mix_norm, false, (const T*)d->g2, (long long)H * E, out, R, H, E, eps, s));
  } else {
    LatentArgs a;
    a.q = d->q; a.dkv = proj + l.s_dkv; a.ld_dkv = l.n_in; a.dkv_norm = theta + l.dkv_norm; a.gate = proj + l.s_g; a.ld_gate = l.n_in;
    a.latent = st.latent; a.ld = l.ld; a.lp = l.lp; a.maxT = c->maxT; a.w_kv = l.w_kv; a.w_ukt = l.w_ukt; a.dp = l.dp; a.oc = d->oc; a.kv = c->kv_exp;
    a.qabs = d->qabs; a.part = c->part; a.part_floats = c->part_floats; a.o = out;
    a.B = B; a.T = Tn; a.first = first; a.heads = H; a.dim = D; a.rot_dim = q.rot_dim; a.rot_dims = q.rot_dims; a.vdim = E; a.kv_rank = q.kv_rank;
    a.scale = q.scale; a.eps = eps; a.freq = l.freq_dev; a.d = d;
    a.dq = proj + l.s_q; a.dq_norm = theta + l.dq_norm; a.cq = d->cq; a.q_rank = q.q_rank; a.qp = l.qp;
    FEMTO_TRY(latent_norms<T>(a, s));
    FEMTO_TRY(rows_linear<T>(d, d->cq, l.qp, l.w_uq, l.qp, d->q, H * (D + q.rot_dim), R, H * (D + q.rot_dim), l.qp, EPI_STORE, s));
    FEMTO_TRY(latent_attention<T>(a, s));
  }
  return rows_linear<T>(d, out, H * E, l.w_o, H * E, d->y, w, R, w, H * E, EPI_STORE, s);
}

// The feed-forward of R rows h: one row each in y, or, with experts, the rows that MoeRows names.
template <typename T>
static int feed_forward(DecoderStack* d, const DecLayer& l, const float* theta, const void* h, void* y, int R, MoeRows& mr, cudaStream_t s) {
  const int w = d->cfg.width;
  const femto_layer_config& q = l.c;
  if (!q.experts) {
    FEMTO_TRY(rows_linear<T>(d, h, w, l.w_gu, w, d->act, l.ffp, R, l.ffp, w, EPI_SWIGLU, s));
    return rows_linear<T>(d, d->act, l.ffp, l.w_down, l.ffp, y, w, R, w, l.ffp, EPI_STORE, s);
  }
  MoeArgs a;
  a.ldz = round_up(q.experts, 4);
  if (sizeof(T) == 2 && R > ROWS_STREAM && (w & 7) == 0 && q.experts <= MOE_ROUTE) a.router = l.w_router;
  else FEMTO_TRY(rows_linear<T>(d, h, w, l.w_router, w, d->moe_z, a.ldz, R, q.experts, w, EPI_F32, s));
  a.z = d->moe_z; a.bias = theta + l.router_bias; a.rows = R; a.experts = q.experts; a.top = q.top; a.width = w;
  a.h = h; a.weight = d->moe_weight; a.expert = d->moe_expert; a.slot = d->moe_slot; a.counts = d->moe_counts; a.groups = d->moe_groups;
  a.lists = d->moe_lists; a.xs = d->moe_x;
  mr.out = d->moe_out; mr.weight = d->moe_weight; mr.top = q.top;
  if constexpr (sizeof(T) == 2) {
    if (R <= ROWS_STREAM && (w & 7) == 0) {
      a.max_lists = std::min(q.experts, R * q.top);
      FEMTO_TRY(moe_choose_few(a, s));
      RowsBatch bt;
      bt.lists = d->moe_lists; bt.max_lists = a.max_lists; bt.x_div = q.top; bt.w = (long long)l.ffp * w;
      FEMTO_TRY(rows_stream((const bf16*)h, w, (const bf16*)l.w_gu, w, d->moe_act, l.ffp, R, l.ffp, w, EPI_RELU2, a.max_lists, bt, s));
      bt.x_div = 1;
      FEMTO_TRY(rows_stream((const bf16*)d->moe_act, l.ffp, (const bf16*)l.w_down, l.ffp, d->moe_out, w, R, w, l.ffp, EPI_STORE, a.max_lists, bt, s));
      return 0;
    }
  }
  a.group_rows = moe_group_rows(R, q.experts, q.top);
  FEMTO_TRY(moe_sort<T>(a, s));
  mr.slot = d->moe_slot;
  GemmArgs g;
  g.ws = d->gemm_ws; g.ws_bytes = d->gemm_ws_bytes; g.status = d->status; g.any_size = true;
  g.groups = d->moe_groups; g.group_rows = a.group_rows; g.n_groups = q.experts;
  g.M = (int)moe_max_slots(R, q.experts, q.top, a.group_rows);
  g.A = d->moe_x; g.lda = w; g.B = l.w_gu; g.ldb = w; g.strideB = (long long)l.ffp * w; g.C = d->moe_act; g.ldc = l.ffp;
  g.N = l.ffp; g.K = w; g.epi = EPI_RELU2;
  FEMTO_TRY(gemm<T>(g, s));
  g.A = d->moe_act; g.lda = l.ffp; g.B = l.w_down; g.ldb = l.ffp; g.C = d->moe_out; g.ldc = w; g.N = w; g.K = l.ffp; g.epi = EPI_STORE;
  return gemm<T>(g, s);
}

// Tokens [t0, t0 + Tn) of every column.
template <typename T>
static int pass_t(DecoderStack* d, femto_kv_cache* c, const float* theta, const int* tokens, int ld_tok, int B, int Tn, float* residuals,
                  cudaStream_t s) {
  typedef DecStream<T> S;
  const int R = B * Tn, w = d->cfg.width, L = d->cfg.n_layer;
  const float eps = d->cfg.norm_eps, m = d->cfg.residual_mult;
  const bool parallel = d->cfg.block == FEMTO_BLOCK_PARALLEL;
  // what follows layer i - 1: the norms of layer i, none after the last
  auto norms_of = [&](int i) {
    NextNorms<T> n;
    if (i == L) return n;
    n.w = theta + d->layers[i].norm1; n.h = (T*)d->hn;
    if (parallel && d->layers[i].c.ff > 0) { n.w2 = theta + d->layers[i].norm2; n.h2 = (T*)d->hn2; }
    return n;
  };
  FEMTO_TRY(S::embed((const T*)d->embed, tokens, ld_tok, B, Tn, d->cfg.index_base, d->cfg.vocab, d->cfg.embed_scale, d->x, norms_of(0), w, eps,
                     d->status, s));
  for (int i = 0; i < L; i++) {
    const DecLayer& l = d->layers[i];
    const bool mlp = l.c.ff > 0;
    const NextNorms<T> next = norms_of(i + 1);
    MoeRows mr;
    FEMTO_TRY(mixer_t<T>(d, c, i, theta, B, Tn, c->len, s));
    if (parallel) {
      if (mlp) FEMTO_TRY(feed_forward<T>(d, l, theta, d->hn2, d->y2, R, mr, s));
      FEMTO_TRY(S::parallel_resid(d->x, (const T*)d->y, mlp && !l.c.experts ? (const T*)d->y2 : nullptr, mr, next, R, w, eps, s));
    } else {
      FEMTO_TRY(S::resid_norm(d->x, (const T*)d->y, theta + l.norm1b, m, mlp ? theta + l.norm2 : next.w, mlp || next.h ? (T*)d->hn : nullptr, R, w, eps, s));
      if (mlp) {
        FEMTO_TRY(feed_forward<T>(d, l, theta, d->hn, d->y, R, mr, s));
        if (l.c.experts) FEMTO_TRY(moe_combine<T>(mr, (T*)d->y, R, w, s));
        FEMTO_TRY(S::resid_norm(d->x, (const T*)d->y, theta + l.norm2b, m, next.w, next.h, R, w, eps, s));
      }
    }
    if (residuals) CUDA_TRY(cudaMemcpyAsync(residuals + (size_t)i * R * w, d->x, 4 * (size_t)R * w, cudaMemcpyDeviceToDevice, s));
  }
  return 0;
}

// Logits of n rows of the residual stream (rows want[0..n), or each column's last) as fp32 [n][vocab].
template <typename T>
static int logits_t(DecoderStack* d, const float* theta, const int* want, int stride, int n, float* out, cudaStream_t s) {
  const int w = d->cfg.width;
  FEMTO_TRY(DecStream<T>::gather_norm(d->x, want, stride, theta + d->off_final, (T*)d->hn, n, w, d->cfg.norm_eps, s));
  RowsOut ro;
  ro.softcap = d->cfg.logit_softcap;
  return rows_linear<T>(d, d->hn, w, d->head, w, out, d->cfg.vocab, n, d->cfg.vocab, w, EPI_F32, s, ro);
}

int decoder_step(femto_handle* h, femto_kv_cache* c, const float* theta, const int* tokens, int B, int T, const int* h_want, int n_want,
                 float* logits_out, float* residuals_out, cudaStream_t s) {
  DecoderStack* d = h->dec;
  if (!d) return femto_fail(FEMTO_ERR_UNSUPPORTED, "the handle's model does not list its layers");
  if (!c || !theta || !tokens || (h_want && (!logits_out || n_want <= 0))) return femto_fail(FEMTO_ERR_ARG, "NULL argument");
  if (c->h != h) return femto_fail(FEMTO_ERR_ARG, "the cache belongs to another handle");
  if (!d->weights_valid) return femto_fail(FEMTO_ERR_STATE, "call femto_refresh_weights before the first step");
  if (B <= 0 || B > c->maxB || T <= 0) return femto_fail(FEMTO_ERR_SHAPE, "step [%d][%d] exceeds the cache's %d columns", B, T, c->maxB);
  if (c->len > 0 && B != c->B) return femto_fail(FEMTO_ERR_SHAPE, "B=%d differs from the %d columns in the cache", B, c->B);
  if ((long long)c->len + T > c->maxT) return femto_fail(FEMTO_ERR_SHAPE, "%d + %d tokens exceed the cache (%d per column)", c->len, T, c->maxT);
  for (int i = 0; i < (h_want ? n_want : 0); i++)
    if (h_want[i] < 0 || h_want[i] >= B * T || (i > 0 && h_want[i] <= h_want[i - 1]))
      return femto_fail(FEMTO_ERR_ARG, "wanted positions must ascend within 0..%d", B * T - 1);
  const int portion = d->cfg.max_rows / B;
  if (residuals_out && T > portion) return femto_fail(FEMTO_ERR_SHAPE, "residuals of %d x %d tokens exceed max_rows", B, T);
  c->B = B;
  for (int t0 = 0; t0 < T; t0 += portion) {
    const int n = std::min(portion, T - t0);
    FEMTO_TRY(d->bf ? pass_t<bf16>(d, c, theta, tokens + t0, T, B, n, residuals_out, s)
                    : pass_t<float>(d, c, theta, tokens + t0, T, B, n, residuals_out, s));
    c->len += n;
    if (!h_want) {
      if (logits_out && t0 + n == T)
        FEMTO_TRY(d->bf ? logits_t<bf16>(d, theta, nullptr, n, B, logits_out, s) : logits_t<float>(d, theta, nullptr, n, B, logits_out, s));
      continue;
    }
    // runs of wanted positions whose logits lie together in the output
    for (int i = 0; i < n_want;) {
      const auto here = [&](int k) { const int t = h_want[k] % T; return t >= t0 && t < t0 + n; };
      if (!here(i)) { i++; continue; }
      std::vector<int> rows;
      int k = i;
      for (; k < n_want && here(k); k++) rows.push_back(h_want[k] / T * n + h_want[k] % T - t0);
      CUDA_TRY(cudaMemcpyAsync(d->want, rows.data(), 4 * rows.size(), cudaMemcpyHostToDevice, s));   // pageable: staged before it returns
      float* out = logits_out + (size_t)i * d->cfg.vocab;
      FEMTO_TRY(d->bf ? logits_t<bf16>(d, theta, d->want, 0, (int)rows.size(), out, s) : logits_t<float>(d, theta, d->want, 0, (int)rows.size(), out, s));
      i = k;
    }
  }
  return 0;
}

// The cache behind femto_kv_cache_*: what a model keeps of the tokens it has seen, for up to maxB columns that have
// all seen the same number of tokens.  The GPT keeps keys and values of every block; a decoder that lists its layers
// keeps, per layer, a recurrent state, the last inputs of short convolutions, or a compressed key/value row per token.
#pragma once
#include <vector>

#include "model.cuh"

struct LayerState {
  float* S = nullptr;          // recurrent state, fp32 [maxB][heads][vdim][dim] (dim contiguous)
  size_t S_bytes = 0;
  void* tail[2] = {nullptr, nullptr};   // last conv - 1 inputs of the convolutions, [maxB][conv - 1][channels] of the compute type;
  size_t tail_bytes = 0;                // a step reads one and writes the other, so blocks of one launch do not race
  int tail_now = 0;
  void* latent = nullptr;      // [maxB][maxT][ld]: latent and rotated key part of every token, compute type
  void* kv = nullptr;          // [maxB][maxT][ld]: keys and values of every token, compute type
  int ld = 0;
};

struct femto_kv_cache {
  femto_handle* h = nullptr;
  int maxB = 0, maxT = 0, B = 0, len = 0;     // len: tokens cached per column (all columns alike)
  char* mem = nullptr;
  std::vector<void*> K, V;                    // GPT, per block: [maxB][maxT][kv] of the compute type
  void* xe_prev = nullptr;                    // GPT: [maxB][d] normalised embedding of the last token (smear)
  void* xe_new = nullptr;                     // GPT: [maxB][d]
  int *tok0 = nullptr, *pos = nullptr, *doc_start = nullptr, *lastpos = nullptr;   // GPT: [maxB]
  float* part = nullptr;                      // split-key partials of the decode attention / split-K of the products
  size_t part_floats = 0;
  std::vector<LayerState> state;              // layer-listing decoders
  void* kv_exp = nullptr;                     // their attention layers: keys and values of one column expanded from the latents
};

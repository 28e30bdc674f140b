// What every decoder of the library has in common: one sequence with a device-resident position and
// token id, the captured one-token graph, the greedy feedback, the chunked prompt pass and the
// capacity checks (decoder_seq.cu).  A model derives from DecoderBase and supplies the launches of one
// token, of one prompt pass and of the output head.
#pragma once

#include "common.cuh"

namespace tlb {

struct DecoderBase {
  int hidden = 0, vocab = 0, max_ctx = 0;
  float* logits = nullptr;   // [vocab] of the last token
  unsigned* d_pos = nullptr;
  int* d_tok = nullptr;      // token consumed by the next forward; overwritten with the result
  int* d_tok_out = nullptr;  // copy of the last result (read back by the host)
  int *h_tok = nullptr, *h_out = nullptr;  // pinned
  // prompt pass: ids of one pass, row indices and logits of the rows a caller asked for
  int* pf_ids = nullptr;
  int pf_id_rows = 0;
  float* want_logits = nullptr;
  long long want_rows = 0;
  cudaGraphExec_t graph = nullptr;
  long long launches_per_token = 0;
  // Host mirror of the device-resident position (captured_decoder::cur_pos of the reference,
  // bench/cuda/qwen_model.h:877-885): every entry point that advances the sequence checks it
  // against the cache capacity before anything is launched.
  long long host_pos = 0;
  long long vocab_total = 0;   // rows of the embedding table (0: unknown, ids are only checked >= 0)

  virtual ~DecoderBase();
  // position, token and logits cells; call once the sizes are set
  int init_base();
  // Enqueue one token (capturable: no sync, no allocation): reads *d_tok and *d_pos, leaves the
  // greedy successor in *d_tok / *d_tok_out and *d_pos + 1.
  virtual int forward(cudaStream_t s) = 0;
  // Before the passes of a prompt: refuse, or size the row-batched scratch for `rows` rows a pass.
  virtual int prefill_begin(int rows, cudaStream_t s) = 0;
  // Most rows of one pass.
  virtual int prefill_rows() const = 0;
  // Run `rows` tokens (device ids) from position `pos`, leaving the rows' last hidden states in place.
  virtual int prefill_pass(const int* d_ids, int rows, int pos, cudaStream_t s) = 0;
  // Logits of `n` rows (host indices) of the pass that just ran, [n, vocab] on the device.
  virtual int head_rows(const int* rows, int n, float* out, cudaStream_t s) = 0;
  // Whether the sequence may be moved to `pos` (a cache that keeps every position allows any).
  virtual int may_seek(long long pos) const { return pos >= 0 && pos < max_ctx; }
};

// TLB_PREFILL_CHUNK, or `dflt`, within [16, 8192]
int prefill_chunk_rows(int dflt);

}  // namespace tlb

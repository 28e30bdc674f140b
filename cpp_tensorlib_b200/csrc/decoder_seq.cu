// The sequence surface every decoder shares (declared in include/tlb200.h as tlb_decoder_*): position
// and token cells, one-token graph, greedy feedback, chunked prompt pass, capacity checks.  The
// structure follows the reference's captured_decoder and prefill_batched (bench/cuda/qwen_model.h:
// 357-442, 791-905).
#include <cstdlib>
#include <string>
#include <vector>

#include "decoder_base.cuh"

namespace tlb {

int launch_argmax(DeviceCtx*, const float*, int, int*, int*, cudaStream_t);

DecoderBase::~DecoderBase() {
  if (graph) cudaGraphExecDestroy(graph);
  cudaFree(logits); cudaFree(d_pos); cudaFree(d_tok); cudaFree(pf_ids); cudaFree(want_logits);
  cudaFreeHost(h_tok);
}

int DecoderBase::init_base() {
  TLB_CUDA(cudaMalloc(&logits, (size_t)vocab * sizeof(float)));
  TLB_CUDA(cudaMalloc(&d_pos, 16));
  TLB_CUDA(cudaMemset(d_pos, 0, 16));
  TLB_CUDA(cudaMalloc(&d_tok, 16));
  TLB_CUDA(cudaMemset(d_tok, 0, 16));
  d_tok_out = d_tok + 1;
  TLB_CUDA(cudaMallocHost(&h_tok, 64));
  h_out = h_tok + 4;
  return TLB_OK;
}

int prefill_chunk_rows(int dflt) {
  int ch = dflt;
  if (const char* e = getenv("TLB_PREFILL_CHUNK")) ch = atoi(e);
  return ch < 16 ? 16 : (ch > 8192 ? 8192 : ch);
}

// The reference's feed() returns false when cur_pos >= max_ctx (bench/cuda/qwen_model.h:879);
// here the refusal is an argument error and nothing is launched.
static int room_for(DecoderBase* d, long long n, const char* who) {
  if (d->host_pos + n > d->max_ctx)
    return set_error(TLB_ERR_ARG, std::string(who) + ": position " + std::to_string(d->host_pos) + " + " +
                                      std::to_string(n) + " token(s) exceeds the cache capacity " +
                                      std::to_string(d->max_ctx));
  return TLB_OK;
}
static int token_ok(DecoderBase* d, long long token, const char* who) {
  if (token < 0 || (d->vocab_total > 0 && token >= d->vocab_total))
    return set_error(TLB_ERR_ARG, std::string(who) + ": token id " + std::to_string(token) +
                                      " outside the embedding table");
  return TLB_OK;
}

}  // namespace tlb

using namespace tlb;

extern "C" {

int tlb_decoder_destroy(void* h) {
  auto* d = (DecoderBase*)h;
  if (!d) return TLB_OK;
  cudaDeviceSynchronize();
  delete d;
  return TLB_OK;
}

int tlb_decoder_logits(void* h, void** logits) {
  auto* d = (DecoderBase*)h;
  TLB_REQUIRE(d && logits, "tlb_decoder_logits: bad arguments");
  *logits = d->logits;
  return TLB_OK;
}
int tlb_decoder_set_pos(void* h, int64_t pos, void* stream) {
  auto* d = (DecoderBase*)h;
  TLB_REQUIRE(d && pos >= 0 && pos < d->max_ctx, "tlb_decoder_set_pos: position outside the cache");
  TLB_REQUIRE(d->may_seek(pos), "tlb_decoder_set_pos: this model's state can only start over or stay where it is");
  d->h_tok[8] = (int)pos;
  TLB_CUDA(cudaMemcpyAsync(d->d_pos, &d->h_tok[8], 4, cudaMemcpyHostToDevice, (cudaStream_t)stream));
  TLB_CUDA(cudaStreamSynchronize((cudaStream_t)stream));
  d->host_pos = pos;
  return TLB_OK;
}
int tlb_decoder_set_token(void* h, int64_t token, void* stream) {
  auto* d = (DecoderBase*)h;
  TLB_REQUIRE(d, "tlb_decoder_set_token: null decoder");
  {
    const int rc = token_ok(d, token, "tlb_decoder_set_token");
    if (rc) return rc;
  }
  d->h_tok[0] = (int)token;
  TLB_CUDA(cudaMemcpyAsync(d->d_tok, d->h_tok, 4, cudaMemcpyHostToDevice, (cudaStream_t)stream));
  TLB_CUDA(cudaStreamSynchronize((cudaStream_t)stream));
  return TLB_OK;
}

// Enqueue one token's launches on `stream` (capturable: no sync, no allocation).
int tlb_decoder_forward(void* h, void* stream) {
  auto* d = (DecoderBase*)h;
  TLB_REQUIRE(d, "tlb_decoder_forward: null decoder");
  int rc = room_for(d, 1, "tlb_decoder_forward");
  if (rc) return rc;
  rc = d->forward((cudaStream_t)stream);
  if (!rc) d->host_pos++;
  return rc;
}
int64_t tlb_decoder_launches_per_token(void* h) {
  auto* d = (DecoderBase*)h;
  return d ? d->launches_per_token : 0;
}

// Capture one forward into an executable graph owned by the decoder
// (qwen_model.h:791-905 captured_decoder::init_).
int tlb_decoder_capture(void* h) {
  auto* d = (DecoderBase*)h;
  TLB_REQUIRE(d, "tlb_decoder_capture: null decoder");
  if (d->graph) { cudaGraphExecDestroy(d->graph); d->graph = nullptr; }
  cudaStream_t s;
  TLB_CUDA(cudaStreamCreateWithFlags(&s, cudaStreamNonBlocking));
  TLB_CUDA(cudaStreamBeginCapture(s, cudaStreamCaptureModeThreadLocal));
  int rc = d->forward(s);
  cudaGraph_t g = nullptr;
  cudaError_t e = cudaStreamEndCapture(s, &g);
  cudaStreamDestroy(s);
  if (rc) { if (g) cudaGraphDestroy(g); return rc; }
  if (e != cudaSuccess) return cuda_fail(e, "cudaStreamEndCapture");
  e = cudaGraphInstantiate(&d->graph, g, 0);
  cudaGraphDestroy(g);
  if (e != cudaSuccess) return cuda_fail(e, "cudaGraphInstantiate");
  return TLB_OK;
}

// Replay the captured token `n` times back to back; the token id feeds back on
// the device (greedy decoding with no host round trip).
int tlb_decoder_run(void* h, int64_t n, void* stream) {
  auto* d = (DecoderBase*)h;
  TLB_REQUIRE(d && d->graph, "tlb_decoder_run: capture the decoder first");
  TLB_REQUIRE(n >= 0, "tlb_decoder_run: negative token count");
  const int rc = room_for(d, n, "tlb_decoder_run");
  if (rc) return rc;
  for (int64_t i = 0; i < n; i++) {
    TLB_CUDA(cudaGraphLaunch(d->graph, (cudaStream_t)stream));
    d->host_pos++;
  }
  return TLB_OK;
}

// End-to-end step with HOST buffers: token id in (host), next token id out (host).
// H2D of the id, one graph replay (or eager launches when not captured), D2H of
// the result, stream synchronised.  token_in < 0 keeps the device-resident token.
int tlb_decoder_step(void* h, const int32_t* token_in, int32_t* token_out, void* stream) {
  auto* d = (DecoderBase*)h;
  TLB_REQUIRE(d && token_out, "tlb_decoder_step: bad arguments");
  cudaStream_t s = (cudaStream_t)stream;
  {
    int rc = room_for(d, 1, "tlb_decoder_step");
    if (!rc && token_in && *token_in >= 0) rc = token_ok(d, *token_in, "tlb_decoder_step");
    if (rc) return rc;
  }
  if (token_in && *token_in >= 0) {
    d->h_tok[0] = *token_in;
    TLB_CUDA(cudaMemcpyAsync(d->d_tok, d->h_tok, 4, cudaMemcpyHostToDevice, s));
  }
  if (d->graph) TLB_CUDA(cudaGraphLaunch(d->graph, s));
  else {
    int rc = d->forward(s);
    if (rc) return rc;
  }
  d->host_pos++;
  TLB_CUDA(cudaMemcpyAsync(d->h_out, d->d_tok_out, 4, cudaMemcpyDeviceToHost, s));
  TLB_CUDA(cudaStreamSynchronize(s));
  *token_out = d->h_out[0];
  return TLB_OK;
}

int tlb_decoder_last_token(void* h, int32_t* token_out, void* stream) {
  auto* d = (DecoderBase*)h;
  TLB_REQUIRE(d && token_out, "tlb_decoder_last_token: bad arguments");
  TLB_CUDA(cudaMemcpyAsync(d->h_out, d->d_tok_out, 4, cudaMemcpyDeviceToHost, (cudaStream_t)stream));
  TLB_CUDA(cudaStreamSynchronize((cudaStream_t)stream));
  *token_out = d->h_out[0];
  return TLB_OK;
}

// The batched prompt pass, in passes of prefill_rows() tokens starting at the decoder's current
// position.  Leaves the caches and the position at pos + T, the greedy next token in the
// device-resident token cell (so tlb_decoder_run continues from there) and in *next_token.
int tlb_decoder_prefill_logits(void* h, const int32_t* tokens, int64_t T, const int32_t* want, int64_t n_want,
                               float* logits_out, int32_t* next_token, void* stream) {
  auto* d = (DecoderBase*)h;
  TLB_REQUIRE(d && tokens && T > 0 && n_want >= 0 && (n_want == 0 || (want && logits_out)),
              "tlb_decoder_prefill: bad arguments");
  cudaStream_t s = (cudaStream_t)stream;
  DeviceCtx* c = nullptr;
  int rc = get_ctx(&c);
  if (rc) return rc;
  unsigned pos0 = 0;
  TLB_CUDA(cudaMemcpyAsync(&pos0, d->d_pos, 4, cudaMemcpyDeviceToHost, s));
  TLB_CUDA(cudaStreamSynchronize(s));
  if ((long long)pos0 + T > d->max_ctx)
    return set_error(TLB_ERR_ARG, "tlb_decoder_prefill: the prompt does not fit the cache");
  for (int64_t i = 0; i < T; i++) {
    rc = token_ok(d, tokens[i], "tlb_decoder_prefill");
    if (rc) return rc;
  }
  for (int64_t i = 0; i < n_want; i++)
    TLB_REQUIRE(want[i] >= 0 && want[i] < T && (i == 0 || want[i] > want[i - 1]),
                "tlb_decoder_prefill_logits: places must increase and lie in the prompt");
  const int CH = d->prefill_rows();
  rc = d->prefill_begin(CH, s);
  if (rc) return rc;
  if (d->pf_id_rows < CH) {
    cudaFree(d->pf_ids);
    d->pf_ids = nullptr;
    TLB_CUDA(cudaMalloc(&d->pf_ids, CH * sizeof(int)));
    d->pf_id_rows = CH;
  }
  int64_t w = 0;
  int last_rows = 0;
  std::vector<int> rows_wanted;
  for (int64_t t0 = 0; t0 < T; t0 += CH) {
    const int rows = (int)((T - t0) < CH ? (T - t0) : CH);
    last_rows = rows;
    TLB_CUDA(cudaMemcpyAsync(d->pf_ids, tokens + t0, (size_t)rows * sizeof(int), cudaMemcpyHostToDevice, s));
    rc = d->prefill_pass(d->pf_ids, rows, (int)(pos0 + t0), s);
    if (rc) return rc;
    rows_wanted.clear();
    const int64_t w0 = w;
    for (; w < n_want && want[w] < t0 + rows; w++) rows_wanted.push_back((int)(want[w] - t0));
    if (rows_wanted.empty()) continue;
    const int n = (int)rows_wanted.size();
    if (d->want_rows < n) {
      cudaFree(d->want_logits);
      d->want_logits = nullptr;
      TLB_CUDA(cudaMalloc(&d->want_logits, (size_t)n * d->vocab * sizeof(float)));
      d->want_rows = n;
    }
    rc = d->head_rows(rows_wanted.data(), n, d->want_logits, s);
    if (rc) return rc;
    TLB_CUDA(cudaMemcpyAsync(logits_out + (size_t)w0 * d->vocab, d->want_logits, (size_t)n * d->vocab * sizeof(float),
                             cudaMemcpyDeviceToHost, s));
  }
  const int last = last_rows - 1;
  rc = d->head_rows(&last, 1, d->logits, s);
  if (!rc) rc = launch_argmax(c, d->logits, d->vocab, d->d_tok, d->d_tok_out, s);
  if (rc) return rc;
  const unsigned newpos = pos0 + (unsigned)T;
  d->h_tok[1] = (int)newpos;
  TLB_CUDA(cudaMemcpyAsync(d->d_pos, &d->h_tok[1], 4, cudaMemcpyHostToDevice, s));
  TLB_CUDA(cudaMemcpyAsync(d->h_out, d->d_tok_out, 4, cudaMemcpyDeviceToHost, s));
  TLB_CUDA(cudaStreamSynchronize(s));
  d->host_pos = (long long)newpos;
  if (next_token) *next_token = d->h_out[0];
  return TLB_OK;
}

int tlb_decoder_prefill(void* h, const int32_t* tokens, int64_t T, int32_t* next_token, void* stream) {
  return tlb_decoder_prefill_logits(h, tokens, T, nullptr, 0, nullptr, next_token, stream);
}

}  // extern "C"

// Native driver of the layer-stack decoder (tlb_stack_* in include/tlb200.h): weights, sequence state,
// scratch, and the launch sequences of one token and of a prompt pass on the shared sequence surface
// (decoder_base.cuh).
//
// One token, five launches a layer (three without a feed-forward), all f32 between the products:
//   [norm1 + input projections of all mixers] -> [all mixers, finished heads] ->
//   [(grouped norm of an ssd or gla mixer) + output projections + residual add] ->
//   [norm2 + gate|up + gated unit] -> [down + residual add]
// Latent attention has four launches of its own beside or instead of the mixers':
//   [query latent's norm + queries] -> [queries to the latent's side, the token's kept row] ->
//   [attention on key ranges] -> [ranges merged, values, gate]
// With the norms behind the sublayers, a sublayer leaves its output alone; the next launch that reads the
// residual adds it up on the way (row_gemv's residual), in one of two buffers in turn.
// Prompt pass with bf16 weights: the same order with tcgen05 products whose operands are the bf16
// rows the norm / finish kernels write, and whose epilogues add the residual or apply the gated unit.
// With f32 weights: the general f32 kernels, one op per launch.
#include <cmath>
#include <cstring>
#include <string>
#include <vector>

#include "decoder_base.cuh"
#include "mixers.cuh"

namespace tlb {

int launch_argmax(DeviceCtx*, const float*, int, int*, int*, cudaStream_t);
int launch_incr_u32(unsigned*, cudaStream_t);

namespace {

int pad8(int n) { return (n + 7) & ~7; }

struct Mat {
  void* W = nullptr;
  int N = 0, K = 0;
  long long ld = 0;
};

struct StackLayer {
  bool has_attn = false;
  AttnP at{};
  RecurP rec[2]{};
  int n_rec = 0, norm_groups[2] = {1, 1};
  int slot[2] = {};              // mixer m: SLOT_ATTN, SLOT_LATENT, or index into rec
  int proj_n = 0, act_n = 0;     // widths of the projected and of the finished row
  int ff = 0;
  float limit = 0.f;
  bool has_latent = false;
  LatentP la{};
  int kv_from = -1;
  Mat uq, ukv;                   // of the latent mixer
  int act = 0;
  const float *norm1 = nullptr, *norm2 = nullptr;
  Mat in, out, gu, down;
};
constexpr int SLOT_ATTN = -1, SLOT_LATENT = -2;
// fewest rows of a prompt pass that expand a latent's keys and values
constexpr int EXPAND_ROWS = 16;

}  // namespace

struct StackDecoder : DecoderBase {
  bool bf16 = true, post_norm = false;
  float eps = 0.f, embed_scale = 1.f, logit_scale = 1.f;
  std::vector<StackLayer> layers;
  Mat embed, head;
  const float* final_norm = nullptr;
  std::vector<void*> owned;
  long long state_bytes = 0;
  int proj_max = 0, act_max = 0, ff_max = 0, conv_max = 0, gate_max = 0, o_max = 0, q_max = 0, chunk = 0;
  int rate_max = 0, qf_max = 0, ql_max = 0;
  // one token
  float *x = nullptr, *x2 = nullptr, *y = nullptr, *proj = nullptr, *act = nullptr, *mb = nullptr;
  float *qv = nullptr, *part = nullptr;      // latent: queries; weighted latents of the key ranges
  void* qa = nullptr;                        // latent: queries on the latent's side
  // prompt pass: rows of pf_rows tokens (hr, actr and ffr in the product's operand type)
  int pf_rows = 0;
  float *xr = nullptr, *projr = nullptr, *orr = nullptr, *tmpr = nullptr, *gath = nullptr;
  float2 *gater = nullptr, *normr = nullptr;
  void *convr = nullptr, *chunkr = nullptr, *hr = nullptr, *qr = nullptr, *actr = nullptr, *ffr = nullptr, *hg = nullptr;
  float *yr = nullptr, *rater = nullptr, *qfr = nullptr, *partr = nullptr;
  void *qlr = nullptr, *qar = nullptr, *exr = nullptr;    // exr: expanded keys and values by slot
  int* idx = nullptr;
  std::vector<void*> pf_owned;

  size_t es() const { return bf16 ? 2 : 4; }
  ~StackDecoder() override {
    for (void* p : owned) cudaFree(p);
    for (void* p : pf_owned) cudaFree(p);
  }
  int alloc(void** p, size_t bytes, std::vector<void*>& pool) {
    TLB_CUDA(cudaMalloc(p, bytes ? bytes : 16));
    pool.push_back(*p);
    TLB_CUDA(cudaMemset(*p, 0, bytes ? bytes : 16));
    return TLB_OK;
  }
  int may_seek(long long pos) const override { return pos == 0 || pos == host_pos; }
  int prefill_rows() const override { return chunk; }
  int forward(cudaStream_t s) override;
  int prefill_begin(int rows, cudaStream_t s) override;
  int prefill_pass(const int* d_ids, int rows, int pos, cudaStream_t s) override;
  int head_rows(const int* rows, int n, float* out, cudaStream_t s) override;
  int ready() const;
  const Mat& out_head() const { return head.W ? head : embed; }
  bool expands(const LatentP& p) const { return bf16 && attn_tiles_eligible(p.qw(), p.Ep); }
  int latent_pass(DeviceCtx* c, const StackLayer& L, int rows, int pos, cudaStream_t s);
  int sublayer_end(DeviceCtx* c, const void* a, long long lda, const Mat& w, const float* norm, int rows, cudaStream_t s);
  int product(DeviceCtx* c, const void* a, long long lda, const Mat& w, float* C, long long ldc, bool add, int rows,
              cudaStream_t s);
};

int StackDecoder::ready() const {
  bool ok = embed.W && final_norm;
  for (auto& L : layers) {
    ok = ok && L.norm1 && L.in.W && L.out.W && (!L.ff || (L.norm2 && L.gu.W && L.down.W));
    if (L.has_attn) ok = ok && L.at.qn && L.at.kn;
    if (L.has_latent) ok = ok && L.la.qn && (L.la.cn || !L.la.owner) && L.uq.W && L.ukv.W;
    for (int i = 0; i < L.n_rec; i++) {
      const RecurP& r = L.rec[i];
      if (r.kind == MIX_GLA) {
        ok = ok && r.norm && r.a_up && r.a_bias;
        continue;
      }
      ok = ok && r.cv.w && r.A_log && r.dt_bias && r.norm && (r.kind == MIX_DELTA || (r.Dskip && r.cv.b));
    }
  }
  return ok ? TLB_OK : set_error(TLB_ERR_STATE, "stack: a weight was never set");
}

int StackDecoder::forward(cudaStream_t s) {
  DeviceCtx* c = nullptr;
  int rc = get_ctx(&c);
  if (!rc) rc = ready();
  if (rc) return rc;
  long long n = 0;
#define RUN(expr)        \
  do {                   \
    rc = (expr);         \
    if (rc) return rc;   \
    n++;                 \
  } while (0)
  auto product1 = [&](const Mat& w, const float* in, float* out, int epi) {
    RowGemv g{};
    g.x = in; g.W = w.W; g.N = w.N; g.K = w.K; g.ldw = w.ld; g.eps = eps; g.y = out; g.epi = epi;
    g.n_groups = 1; g.nscale = 1.f;
    return g;
  };
  auto normed = [&](RowGemv& g, const float* nw, int n_off, int n_len, int groups, float scale) {
    g.nw = nw; g.n_off = n_off; g.n_len = n_len; g.n_groups = groups; g.nscale = scale;
  };
  auto gemv = [&](const RowGemv& g) { return row_gemv_launch(c, g, bf16, s); };
  float *cur = x, *alt = x2;
  const float* pending = nullptr;   // norm of the sublayer output in y that the residual still lacks
  auto from_residual = [&](const Mat& w, float* out, int epi) {
    RowGemv g = product1(w, cur, out, epi);
    if (pending) {
      g.x = y; g.res = cur; g.rn = pending; g.xout = alt;
      float* t = cur;
      cur = alt;
      alt = t;
      pending = nullptr;
    }
    return g;
  };
  RUN(embed_scaled_launch(embed.W, d_tok, x, hidden, embed.ld, embed_scale, 1, bf16, s));
  for (auto& L : layers) {
    RowGemv g = from_residual(L.in, proj, 0);
    if (!post_norm) normed(g, L.norm1, 0, hidden, 1, 1.f);
    RUN(gemv(g));
    if (L.has_attn || L.n_rec)
      RUN(mixers_decode_launch(L.has_attn ? &L.at : nullptr, L.rec, L.n_rec, proj, act, d_pos, bf16, s));
    if (L.has_latent) {
      g = product1(L.uq, proj + L.la.oq, qv, 0);
      normed(g, L.la.qn, 0, L.la.Q, 1, 1.f);
      RUN(gemv(g));
      RUN(latent_absorb_launch(L.la, qv, L.uq.N, proj, qa, 1, d_pos, 0, bf16, s));
      RUN(latent_attend_launch(L.la, qa, part, 1, L.la.splits, d_pos, 0, bf16, s));
      RUN(latent_fold_launch(L.la, part, L.la.splits, proj, L.proj_n, act, L.act_n, 1, d_pos, 0, bf16, false, s));
    }
    g = product1(L.out, act, post_norm ? y : cur, post_norm ? 0 : 1);
    for (int i = 0; i < L.n_rec; i++) {   // the norm of an ssd or gla mixer runs in front of the output projection
      const RecurP& r = L.rec[i];
      if (r.kind == MIX_DELTA) continue;
      normed(g, r.norm, r.oa, r.H * r.E, L.norm_groups[i], r.out_scale);
      if (r.kind == MIX_GLA) g.gate = proj + r.og;
    }
    RUN(gemv(g));
    if (post_norm) pending = L.norm1;
    if (L.ff) {
      g = from_residual(L.gu, mb, L.act ? 3 : 2);
      g.limit = L.limit;
      if (!post_norm) normed(g, L.norm2, 0, hidden, 1, 1.f);
      RUN(gemv(g));
      RUN(gemv(product1(L.down, mb, post_norm ? y : cur, post_norm ? 0 : 1)));
      if (post_norm) pending = L.norm2;
    }
  }
  RowGemv g = from_residual(out_head(), logits, 0);
  g.xout = nullptr;
  normed(g, final_norm, 0, hidden, 1, logit_scale);
  RUN(gemv(g));
  RUN(launch_argmax(c, logits, vocab, d_tok, d_tok_out, s));
  RUN(launch_incr_u32(d_pos, s));
#undef RUN
  launches_per_token = n;
  return TLB_OK;
}

int StackDecoder::prefill_begin(int rows, cudaStream_t s) {
  int rc = ready();
  if (rc) return rc;
  if (pf_rows >= rows) return TLB_OK;
  TLB_CUDA(cudaStreamSynchronize(s));
  for (void* p : pf_owned) cudaFree(p);
  pf_owned.clear();
  pf_rows = 0;
  const size_t R = rows;
  auto get = [&](auto** p, size_t bytes) { if (!rc) rc = alloc((void**)p, bytes, pf_owned); };
  get(&xr, R * hidden * 4);
  get(&projr, R * proj_max * 4);
  get(&convr, R * conv_max * 4);
  get(&orr, R * o_max * 4);
  get(&gater, R * gate_max * sizeof(float2));
  get(&normr, R * gate_max * sizeof(float2));
  size_t cb = 0;
  for (auto& L : layers)
    for (int i = 0; i < L.n_rec; i++) {
      const RecurP& r = L.rec[i];
      size_t n = 0;
      if (r.kind == MIX_GLA) n = bf16 && gla_chunk_eligible(r) ? gla_chunk_scratch_bytes(r, rows) : 0;
      else if (bf16 && recur_chunk_eligible(r)) n = recur_chunk_scratch_bytes(r, rows);
      cb = n > cb ? n : cb;
    }
  get(&chunkr, cb);
  get(&gath, R * hidden * 4);
  get(&hr, R * pad8(hidden) * es());
  get(&hg, R * pad8(hidden) * es());
  get(&qr, R * q_max * es());
  get(&actr, R * act_max * es());
  get(&ffr, R * pad8(ff_max) * es());
  get(&idx, R * sizeof(int));
  size_t part_floats = 0, ab = 0, eb = 0;
  for (auto& L : layers) {
    if (!L.has_latent) continue;
    const LatentP& p = L.la;
    const int n = expands(p) && rows >= EXPAND_ROWS ? EXPAND_ROWS : rows;   // most rows of the general form
    for (int r = 1; r <= n; r++) {
      const size_t f = latent_part_floats(p, r, latent_splits(p, r));
      part_floats = f > part_floats ? f : part_floats;
    }
    const size_t a = (size_t)n * p.H * p.row() * es(), e = (size_t)p.ring * p.H * (p.Dp + p.Ep) * 2;
    ab = a > ab ? a : ab;
    if (expands(p)) eb = e > eb ? e : eb;
  }
  get(&partr, part_floats * 4);
  get(&qar, ab);
  get(&exr, eb);
  get(&qfr, R * qf_max * 4);
  get(&qlr, R * ql_max * es());
  get(&rater, R * rate_max * 4);
  if (post_norm) get(&yr, R * hidden * 4);
  if (!bf16) get(&tmpr, R * (size_t)(2 * ff_max > hidden ? 2 * ff_max : hidden) * 4);
  if (!rc) pf_rows = rows;
  return rc;
}

// C[rows, N] = (C +) a . W^T
int StackDecoder::product(DeviceCtx* c, const void* a, long long lda, const Mat& w, float* C, long long ldc, bool add,
                          int rows, cudaStream_t s) {
  if (bf16) return gemm_bf16_tc_launch(c, a, lda, w.W, w.ld, C, ldc, nullptr, 0, rows, w.N, w.K, add ? 1 : 0, 0.f, s);
  int rc = tlb_gemm_f32((const float*)a, lda, 0, (const float*)w.W, w.ld, 1, add ? tmpr : C, rows, w.N, w.K, 1.f, 0.f, s);
  if (!rc && add) rc = tlb_binary(TLB_OP_ADD, C, tmpr, C, (int64_t)rows * w.N, 1.f, 0.f, s);
  return rc;
}

// Latent attention of a pass: the projected rows are there, the finished heads go to actr.
int StackDecoder::latent_pass(DeviceCtx* c, const StackLayer& L, int rows, int pos, cudaStream_t s) {
  const LatentP& p = L.la;
  int rc = latent_prep_launch(p, projr, L.proj_n, rows, pos, qlr, bf16, s);
  if (!rc) rc = product(c, qlr, p.Qp, L.uq, qfr, L.uq.N, false, rows, s);
  if (rc) return rc;
  if (!expands(p) || rows < EXPAND_ROWS) {
    const int splits = latent_splits(p, rows);
    rc = latent_absorb_launch(p, qfr, L.uq.N, nullptr, qar, rows, nullptr, pos, bf16, s);
    if (!rc) rc = latent_attend_launch(p, qar, partr, rows, splits, nullptr, pos, bf16, s);
    if (!rc) rc = latent_fold_launch(p, partr, splits, projr, L.proj_n, actr, L.act_n, rows, nullptr, pos, bf16, bf16, s);
    return rc;
  }
  rc = latent_q_rows_launch(p, qfr, L.uq.N, qr, rows, pos, s);
  if (rc) return rc;
  // keys and values of the rows in sight, in the slots of the latents they come from
  const int n = L.ukv.N, first = pos + rows > p.ring ? 0 : (pos + 1 > p.window ? pos + 1 - p.window : 0);
  const int last = pos + rows > p.ring ? p.ring : pos + rows;
  const __nv_bfloat16* kept = (const __nv_bfloat16*)p.rows;
  __nv_bfloat16* ex = (__nv_bfloat16*)exr;
  rc = gemm_bf16_tc_launch(c, kept + (size_t)first * p.row(), p.row(), L.ukv.W, L.ukv.ld, nullptr, 0, ex + (size_t)first * n,
                           n, last - first, n, p.C, 3, 0.f, s);
  if (rc) return rc;
  AttnTiles t{};
  t.q = qr; t.q_row = (long long)p.H * p.qw(); t.q_head = p.qw();
  t.k = ex; t.k_row = n; t.k_head = p.Dp; t.kw = p.Dp;
  t.k2 = kept + p.Cp; t.k2_row = p.row(); t.k2w = p.Rp;
  t.v = ex + (size_t)p.H * p.Dp; t.v_row = n; t.v_head = p.Ep; t.vw = p.Ep;
  t.H = p.H; t.R = 1; t.E = p.E;
  t.window = p.window; t.keep = 0; t.ring = p.ring;
  t.scale = p.scale; t.out_scale = p.out_scale;
  t.gate = p.og >= 0 ? projr + p.og : nullptr; t.gate_row = L.proj_n;
  return attn_tiles_launch(t, (__nv_bfloat16*)actr + p.oa, L.act_n, rows, pos, s);
}

// The last product of a sublayer and the residual: added in the product's epilogue, or normed first (the
// next product's operand hr comes with it).
int StackDecoder::sublayer_end(DeviceCtx* c, const void* a, long long lda, const Mat& w, const float* norm, int rows,
                               cudaStream_t s) {
  if (!post_norm) return product(c, a, lda, w, xr, hidden, true, rows, s);
  const int rc = product(c, a, lda, w, yr, hidden, false, rows, s);
  return rc ? rc : residual_rows_launch(xr, yr, norm, hr, pad8(hidden), hidden, eps, rows, bf16, s);
}

int StackDecoder::prefill_pass(const int* d_ids, int rows, int pos, cudaStream_t s) {
  DeviceCtx* c = nullptr;
  int rc = get_ctx(&c);
  if (rc) return rc;
#define PF(expr) do { rc = (expr); if (rc) return rc; } while (0)
  const int E8 = pad8(hidden);
  PF(embed_scaled_launch(embed.W, d_ids, xr, hidden, embed.ld, embed_scale, rows, bf16, s));
  if (post_norm) PF(residual_rows_launch(xr, nullptr, nullptr, hr, E8, hidden, eps, rows, bf16, s));
  for (auto& L : layers) {
    if (!post_norm) PF(rms_rows_launch(xr, hidden, L.norm1, hr, E8, hidden, eps, 1.f, rows, bf16, s));
    PF(product(c, hr, E8, L.in, projr, L.proj_n, false, rows, s));
    if (L.has_attn) {
      PF(attn_rows_prep_launch(L.at, projr, L.proj_n, rows, pos, qr, bf16, s));
      if (bf16 && attn_window_eligible(L.at))
        PF(attn_window_launch(L.at, qr, projr, L.proj_n, actr, L.act_n, rows, pos, s));
      else
        PF(attn_rows_launch(L.at, qr, projr, L.proj_n, actr, L.act_n, rows, pos, bf16, s));
    }
    if (L.has_latent) PF(latent_pass(c, L, rows, pos, s));
    for (int i = 0; i < L.n_rec; i++) {
      const RecurP& r = L.rec[i];
      if (r.kind == MIX_GLA) {
        PF(gla_rates_launch(r, projr, L.proj_n, rater, rows, s));
        if (bf16 && gla_chunk_eligible(r)) PF(gla_chunk_launch(r, projr, L.proj_n, rater, chunkr, orr, rows, pos, s));
        else PF(recur_rows_scan_launch(r, projr, L.proj_n, rater, orr, rows, pos, s));
        PF(recur_rows_finish_launch(r, orr, nullptr, false, projr, L.proj_n, actr, L.act_n, 1, rows, bf16, s));
        continue;
      }
      const bool chunks = bf16 && recur_chunk_eligible(r);
      PF(recur_rows_conv_launch(r, projr, L.proj_n, rows, pos, convr, gater, normr, chunks, s));
      if (chunks) PF(recur_chunk_launch(r, convr, gater, normr, chunkr, orr, rows, pos, s));
      else PF(recur_rows_scan_launch(r, (const float*)convr, r.cv.C, gater, orr, rows, pos, s));
      PF(recur_rows_finish_launch(r, orr, convr, chunks, projr, L.proj_n, actr, L.act_n, L.norm_groups[i], rows, bf16, s));
    }
    PF(sublayer_end(c, actr, L.act_n, L.out, L.norm1, rows, s));
    if (!L.ff) continue;
    const int F8 = bf16 ? pad8(L.ff) : L.ff;
    if (!post_norm) PF(rms_rows_launch(xr, hidden, L.norm2, hr, E8, hidden, eps, 1.f, rows, bf16, s));
    if (bf16) {
      PF(gemm_bf16_tc_launch(c, hr, E8, L.gu.W, L.gu.ld, nullptr, 0, ffr, F8, rows, L.gu.N, L.gu.K, L.act ? 4 : 2, L.limit, s));
    } else {
      PF(tlb_gemm_f32((const float*)hr, E8, 0, (const float*)L.gu.W, L.gu.ld, 1, tmpr, rows, L.gu.N, L.gu.K, 1.f, 0.f, s));
      if (L.act) PF(relu2_rows_launch(tmpr, (float*)ffr, L.ff, rows, s));
      else PF(glu_rows_launch(tmpr, (float*)ffr, L.ff, L.limit, rows, s));
    }
    PF(sublayer_end(c, ffr, F8, L.down, L.norm2, rows, s));
  }
#undef PF
  return TLB_OK;
}

int StackDecoder::head_rows(const int* rows, int n, float* out, cudaStream_t s) {
  DeviceCtx* c = nullptr;
  int rc = get_ctx(&c);
  if (rc) return rc;
  if (n == 1) {   // the projection's own norm and weight stream
    RowGemv g{};
    const Mat& w = out_head();
    g.x = xr + (size_t)rows[0] * hidden; g.W = w.W; g.N = w.N; g.K = w.K; g.ldw = w.ld;
    g.nw = final_norm; g.n_len = hidden; g.n_groups = 1; g.eps = eps; g.nscale = logit_scale; g.y = out;
    return row_gemv_launch(c, g, bf16, s);
  }
  TLB_CUDA(cudaMemcpyAsync(idx, rows, (size_t)n * sizeof(int), cudaMemcpyHostToDevice, s));
  rc = gather_rows_launch(xr, idx, gath, hidden, n, s);
  if (!rc) rc = rms_rows_launch(gath, hidden, final_norm, hg, pad8(hidden), hidden, eps, logit_scale, n, bf16, s);
  if (!rc) rc = product(c, hg, pad8(hidden), out_head(), out, vocab, false, n, s);
  return rc;
}

static int max_i(int a, int b) { return a > b ? a : b; }

// angular frequencies of a rotation, in two floats each
static int rotation_table(StackDecoder* d, float base, int dims, const float2** out) {
  std::vector<float2> f(max_i(1, dims / 2));
  for (int i = 0; i < dims / 2; i++) {
    const double w = pow((double)base, -2.0 * i / dims);
    f[i].x = (float)w;
    f[i].y = (float)(w - (double)f[i].x);
  }
  float2* df = nullptr;
  const int rc = d->alloc((void**)&df, f.size() * sizeof(float2), d->owned);
  if (rc) return rc;
  TLB_CUDA(cudaMemcpy(df, f.data(), f.size() * sizeof(float2), cudaMemcpyHostToDevice));
  *out = df;
  return TLB_OK;
}

// Kept rows of the latent layers: an owner keeps what the widest window of its readers and one pass need.
static int build_latents(StackDecoder* d, DeviceCtx* c) {
  int rc = TLB_OK;
  size_t part = 0, qa = 0, qv = 0;
  for (auto& L : d->layers)
    if (L.has_latent && !L.la.owner) {
      LatentP& o = d->layers[L.kv_from].la;
      o.ring = max_i(o.ring, L.la.window);
    }
  for (auto& L : d->layers) {
    if (!L.has_latent) continue;
    LatentP& p = L.la;
    if (p.owner) {
      const int need = max_i(p.ring, p.window) + d->chunk;
      p.ring = need < d->max_ctx ? need : d->max_ctx;
      const size_t bytes = (size_t)p.ring * p.row() * d->es();
      if (!rc) rc = d->alloc(&p.rows, bytes, d->owned);
      d->state_bytes += bytes;
    } else {
      p.rows = d->layers[L.kv_from].la.rows;
      p.ring = d->layers[L.kv_from].la.ring;
    }
    const int units = (p.H + 15) / 16, tiles = (p.window + 63) / 64;
    p.splits = max_i(1, c->sm_count / units);
    if (p.splits > 64) p.splits = 64;
    if (p.splits > tiles) p.splits = tiles;
    const size_t f = latent_part_floats(p, 1, p.splits), a = (size_t)p.H * p.row() * d->es(), q = (size_t)p.H * p.qw();
    part = f > part ? f : part;
    qa = a > qa ? a : qa;
    qv = q > qv ? q : qv;
    d->q_max = max_i(d->q_max, p.H * p.qw());
    d->qf_max = max_i(d->qf_max, p.H * p.qw());
    d->ql_max = max_i(d->ql_max, p.Qp);
  }
  if (!rc && part) rc = d->alloc((void**)&d->part, part * 4, d->owned);
  if (!rc && qa) rc = d->alloc(&d->qa, qa, d->owned);
  if (!rc && qv) rc = d->alloc((void**)&d->qv, qv * 4, d->owned);
  return rc;
}

static int build(StackDecoder* d, const tlb_stack_cfg* cfg, const tlb_layer_cfg* ls) {
  DeviceCtx* c = nullptr;
  int rc = get_ctx(&c);
  if (rc) return rc;
  d->hidden = cfg->width; d->vocab = cfg->vocab; d->max_ctx = cfg->max_ctx; d->vocab_total = cfg->vocab;
  d->bf16 = !cfg->f32; d->eps = cfg->eps; d->embed_scale = cfg->embed_scale;
  d->post_norm = cfg->post_norm != 0; d->logit_scale = cfg->logit_scale;
  TLB_REQUIRE(d->hidden > 0 && d->vocab > 0 && d->max_ctx > 0 && cfg->n_layers > 0, "tlb_stack_create: bad sizes");
  const int rows = prefill_chunk_rows(4096);
  d->chunk = rows < d->max_ctx ? rows : d->max_ctx;
  d->layers.resize(cfg->n_layers);
  for (int l = 0; l < cfg->n_layers; l++) {
    const tlb_layer_cfg& lc = ls[l];
    StackLayer& L = d->layers[l];
    TLB_REQUIRE(lc.n_mixers >= 1 && lc.n_mixers <= 2 && lc.ff >= 0, "tlb_stack_create: bad layer");
    L.ff = lc.ff; L.limit = lc.limit; L.act = lc.act;
    TLB_REQUIRE(lc.act == 0 || lc.act == 1, "tlb_stack_create: unknown feed-forward");
    for (int m = 0; m < lc.n_mixers; m++) {
      const tlb_mixer_cfg& k = lc.mixer[m];
      const int H = k.heads, G = k.kv_heads, D = k.dim, E = k.vdim;
      TLB_REQUIRE(H > 0 && G > 0 && H % G == 0 && D > 0 && E > 0, "tlb_stack_create: bad head counts or widths");
      auto take = [&](int n) { const int o = L.proj_n; L.proj_n += pad8(n); return o; };
      const int oa = L.act_n;
      L.act_n += pad8(H * E);
      if (k.kind == TLB_MIX_ATTN) {
        TLB_REQUIRE(!L.has_attn, "tlb_stack_create: one attention a layer");
        TLB_REQUIRE(E <= 2 * MX_THREADS && D <= 1024, "tlb_stack_create: attention head too wide");
        TLB_REQUIRE(k.window > 0 && k.keep_first >= 0 && k.rot_dims >= 0 && k.rot_dims <= D && k.rot_dims % 2 == 0,
                    "tlb_stack_create: bad window or rotation");
        L.has_attn = true;
        L.slot[m] = SLOT_ATTN;
        AttnP& p = L.at;
        p.H = H; p.G = G; p.D = D; p.E = E; p.Dp = pad8(D); p.Ep = p.Vs = pad8(E);
        p.window = k.window < d->max_ctx ? k.window : d->max_ctx;
        p.keep = k.keep_first < d->max_ctx ? k.keep_first : d->max_ctx;
        p.pairs = k.rot_dims / 2; p.scale = k.scale; p.eps = d->eps; p.out_scale = k.out_scale; p.oa = oa;
        p.oq = take(H * D); p.ok = take(G * D); p.ov = take(G * E); p.og = take(H * E);
        // keys a pass can reach: the window in front of its first row and the pass itself
        const int span = p.window + d->chunk, rest = max_i(1, d->max_ctx - p.keep);
        p.ring = span < rest ? span : rest;
        p.cap = p.keep + p.ring;
        const size_t kb = (size_t)G * p.cap * p.Dp * d->es(), vb = (size_t)G * p.cap * p.Ep * d->es();
        if (!rc) rc = d->alloc(&p.K, kb, d->owned);
        if (!rc) rc = d->alloc(&p.V, vb, d->owned);
        d->state_bytes += kb + vb;
        const int R = H / G;
        p.hb = (R + 7) / 8; p.hpb = (R + p.hb - 1) / p.hb;
        const int units = G * p.hb, most = p.window + p.keep;
        p.splits = max_i(1, (2 * c->sm_count) / units);
        if (p.splits > (most + 63) / 64) p.splits = (most + 63) / 64;
        if (p.splits > MX_TK) p.splits = MX_TK;
        if (!rc) rc = d->alloc((void**)&p.part, units * attn_part_floats(p) * 4, d->owned);
        if (!rc) rc = d->alloc((void**)&p.counters, (size_t)units * sizeof(int), d->owned);
        if (!rc) rc = rotation_table(d, k.rot_base, k.rot_dims, &p.inv_freq);
        if (rc) return rc;
        d->q_max = max_i(d->q_max, H * p.Dp);
      } else if (k.kind == TLB_MIX_LATENT) {
        TLB_REQUIRE(!L.has_latent, "tlb_stack_create: one latent attention a layer");
        TLB_REQUIRE(k.q_rank > 0 && k.kv_rank > 0 && k.kv_rank <= 8192 && D <= 1024, "tlb_stack_create: latent too wide");
        TLB_REQUIRE(k.window >= 0 && k.rot_dims >= 0 && k.rot_dims <= 2 * MX_PAIRS && k.rot_dims % 2 == 0,
                    "tlb_stack_create: bad window or rotation");
        L.has_latent = true;
        L.slot[m] = SLOT_LATENT;
        L.kv_from = k.kv_from;
        LatentP& p = L.la;
        p.H = H; p.D = D; p.R = k.rot_dims; p.E = E; p.Q = k.q_rank; p.C = k.kv_rank;
        p.Dp = pad8(D); p.Rp = pad8(p.R); p.Ep = pad8(E); p.Qp = pad8(p.Q); p.Cp = pad8(p.C);
        p.window = k.window > 0 && k.window < d->max_ctx ? k.window : d->max_ctx;
        p.owner = k.kv_from < 0;
        p.scale = k.scale; p.eps = d->eps; p.out_scale = k.out_scale; p.oa = oa;
        if (!p.owner) {
          TLB_REQUIRE(k.kv_from < l && d->layers[k.kv_from].has_latent && d->layers[k.kv_from].la.owner,
                      "tlb_stack_create: kv_from must name an earlier latent layer that keeps its own rows");
          const LatentP& o = d->layers[k.kv_from].la;
          TLB_REQUIRE(o.C == p.C && o.R == p.R, "tlb_stack_create: layers that share a latent have one width of it");
        }
        p.oq = take(p.Q);
        if (p.owner) { p.oc = take(p.C); take(p.R); }
        p.og = k.gate ? take(H * E) : -1;
        if (!rc) rc = rotation_table(d, k.rot_base, p.R, &p.inv_freq);
        if (rc) return rc;
      } else if (k.kind == TLB_MIX_GLA) {
        TLB_REQUIRE(D <= 1024 && k.rank > 0 && k.tau > 0.f, "tlb_stack_create: bad gla sizes");
        for (int i = 0; i < L.n_rec; i++)
          TLB_REQUIRE(L.rec[i].kind == MIX_DELTA, "tlb_stack_create: one ssd or gla mixer a layer");
        L.slot[m] = L.n_rec;
        RecurP& r = L.rec[L.n_rec];
        L.norm_groups[L.n_rec] = H;
        r.kind = k.kind; r.H = r.G = H; r.D = D; r.E = E; r.eps = d->eps; r.out_scale = k.out_scale; r.oa = oa;
        r.rank = k.rank; r.tau = k.tau;
        r.cq = take(H * D); r.ck = take(H * D); r.cvv = take(H * E); r.og = take(H * E); r.ob = take(k.rank);
        const size_t sb = (size_t)H * D * E * 4;
        if (!rc) rc = d->alloc((void**)&r.S, sb, d->owned);
        if (rc) return rc;
        d->state_bytes += sb;
        d->o_max = max_i(d->o_max, H * E);
        d->rate_max = max_i(d->rate_max, H * D);
        L.n_rec++;
      } else if (k.kind == TLB_MIX_DELTA || k.kind == TLB_MIX_SSD) {
        TLB_REQUIRE(D <= 1024, "tlb_stack_create: recurrent state too wide");
        TLB_REQUIRE(k.conv >= 1, "tlb_stack_create: a convolution has at least one tap");
        L.slot[m] = L.n_rec;
        RecurP& r = L.rec[L.n_rec];
        L.norm_groups[L.n_rec] = k.kind == TLB_MIX_SSD ? k.norm_groups : 1;
        r.kind = k.kind; r.H = H; r.G = G; r.D = D; r.E = E; r.eps = d->eps; r.out_scale = k.out_scale; r.oa = oa;
        r.cv.taps = k.conv;
        if (k.kind == TLB_MIX_DELTA) {
          r.cv.off = take(G * D);
          take(G * D); take(H * E);
          r.cq = 0; r.ck = pad8(G * D); r.cvv = 2 * pad8(G * D);
          r.cv.C = r.cvv + pad8(H * E);
          r.og = take(H * E); r.ob = take(H); r.oa_ = take(H);
        } else {
          TLB_REQUIRE(k.norm_groups > 0 && (H * E) % k.norm_groups == 0, "tlb_stack_create: bad norm groups");
          TLB_REQUIRE(L.n_rec == 0 || L.rec[0].kind == MIX_DELTA, "tlb_stack_create: one ssd or gla mixer a layer");
          r.og = take(H * E);
          r.cv.C = pad8(H * E + 2 * G * D);
          r.cv.off = take(H * E + 2 * G * D);
          r.cvv = 0; r.ck = H * E; r.cq = H * E + G * D;
          r.ob = take(H); r.oa_ = r.ob;
        }
        const size_t sb = (size_t)H * D * E * 4, rb = (size_t)r.cv.taps * r.cv.C * 4;
        if (!rc) rc = d->alloc((void**)&r.S, sb, d->owned);
        if (!rc) rc = d->alloc((void**)&r.cv.ring, rb, d->owned);
        if (rc) return rc;
        d->state_bytes += sb + rb;
        d->conv_max = max_i(d->conv_max, r.cv.C);
        d->gate_max = max_i(d->gate_max, H);
        d->o_max = max_i(d->o_max, H * E);
        L.n_rec++;
      } else {
        return set_error(TLB_ERR_ARG, "tlb_stack_create: unknown mixer");
      }
    }
    d->proj_max = max_i(d->proj_max, L.proj_n);
    d->act_max = max_i(d->act_max, L.act_n);
    d->ff_max = max_i(d->ff_max, L.ff);
  }
  if (!rc) rc = build_latents(d, c);
  if (!rc) rc = d->alloc((void**)&d->x, (size_t)d->hidden * 4, d->owned);
  if (!rc) rc = d->alloc((void**)&d->x2, (size_t)d->hidden * 4, d->owned);
  if (!rc) rc = d->alloc((void**)&d->y, (size_t)d->hidden * 4, d->owned);
  if (!rc) rc = d->alloc((void**)&d->proj, (size_t)d->proj_max * 4, d->owned);
  if (!rc) rc = d->alloc((void**)&d->act, (size_t)d->act_max * 4, d->owned);
  if (!rc) rc = d->alloc((void**)&d->mb, (size_t)(d->ff_max + 8) * 4, d->owned);
  if (!rc) rc = d->init_base();
  if (!rc) TLB_CUDA(cudaDeviceSynchronize());
  return rc;
}

}  // namespace tlb

using namespace tlb;

static StackDecoder* as_stack(void* h) { return dynamic_cast<StackDecoder*>((DecoderBase*)h); }

extern "C" {

int tlb_stack_create(const tlb_stack_cfg* cfg, const tlb_layer_cfg* layers, void** out) {
  TLB_REQUIRE(cfg && layers && out, "tlb_stack_create: bad arguments");
  auto* d = new StackDecoder();
  const int rc = build(d, cfg, layers);
  if (rc) { delete d; return rc; }
  *out = static_cast<DecoderBase*>(d);
  return TLB_OK;
}

int tlb_stack_set_matrix(void* h, int64_t layer, int which, const void* w, int64_t rows, int64_t cols) {
  StackDecoder* d = as_stack(h);
  TLB_REQUIRE(d && w && rows > 0 && cols > 0, "tlb_stack_set_matrix: bad arguments");
  Mat* m = nullptr;
  int64_t N = 0, K = 0;
  if (which == 4 || which == 5) { m = which == 4 ? &d->embed : &d->head; N = d->vocab; K = d->hidden; }
  else {
    TLB_REQUIRE(layer >= 0 && layer < (int64_t)d->layers.size(), "tlb_stack_set_matrix: layer out of range");
    StackLayer& L = d->layers[layer];
    if (which == 0) { m = &L.in; N = L.proj_n; K = d->hidden; }
    else if (which == 1) { m = &L.out; N = d->hidden; K = L.act_n; }
    else if (which == 2) { m = &L.gu; N = L.act ? L.ff : 2 * L.ff; K = d->hidden; }
    else if (which == 3) { m = &L.down; N = d->hidden; K = L.ff; }
    else if (which >= 16 && which < 32) {
      const int mixer = which & 7;
      TLB_REQUIRE(mixer < 2 && L.has_latent && L.slot[mixer] == SLOT_LATENT, "tlb_stack_set_matrix: not a latent mixer");
      const LatentP& p = L.la;
      if (which < 24) { m = &L.uq; N = (int64_t)p.H * p.qw(); K = p.Q; }
      else { m = &L.ukv; N = (int64_t)p.H * (p.Dp + p.Ep); K = p.C; }
    }
    else return set_error(TLB_ERR_ARG, "tlb_stack_set_matrix: unknown matrix id");
  }
  TLB_REQUIRE(rows == N && cols == K, "tlb_stack_set_matrix: shape does not match the layer");
  const size_t es = d->es(), ld = (size_t)(cols + 7) & ~(size_t)7;
  if (!m->W) {
    const int rc = d->alloc(&m->W, (size_t)rows * ld * es, d->owned);
    if (rc) return rc;
  }
  m->N = (int)rows; m->K = (int)cols; m->ld = (long long)ld;
  if (which >= 16) {
    LatentP& p = d->layers[layer].la;
    (which < 24 ? p.uq : p.ukv) = m->W;
  }
  TLB_CUDA(cudaMemcpy2D(m->W, ld * es, w, (size_t)cols * es, (size_t)cols * es, (size_t)rows, cudaMemcpyHostToDevice));
  return TLB_OK;
}

int tlb_stack_set_vector(void* h, int64_t layer, int mixer, int which, const float* v, int64_t n) {
  StackDecoder* d = as_stack(h);
  TLB_REQUIRE(d && v && n > 0, "tlb_stack_set_vector: bad arguments");
  const float** dst = nullptr;
  int64_t want = 0;
  if (which == 2) { dst = &d->final_norm; want = d->hidden; }
  else {
    TLB_REQUIRE(layer >= 0 && layer < (int64_t)d->layers.size(), "tlb_stack_set_vector: layer out of range");
    StackLayer& L = d->layers[layer];
    if (which == 0) { dst = &L.norm1; want = d->hidden; }
    else if (which == 1) { dst = &L.norm2; want = d->hidden; }
    else {
      TLB_REQUIRE(mixer >= 0 && mixer < 2 && mixer < L.n_rec + L.has_attn + L.has_latent, "tlb_stack_set_vector: no such mixer");
      if (L.slot[mixer] == SLOT_LATENT) {
        if (which == 10) { dst = &L.la.qn; want = L.la.Q; }
        else if (which == 11) { dst = &L.la.cn; want = L.la.C; }
      } else if (L.slot[mixer] == SLOT_ATTN) {
        if (which == 10) { dst = &L.at.qn; want = (int64_t)L.at.H * L.at.D; }
        else if (which == 11) { dst = &L.at.kn; want = (int64_t)L.at.G * L.at.D; }
      } else {
        RecurP& r = L.rec[L.slot[mixer]];
        if (which == 12) { dst = &r.norm; want = r.kind == MIX_DELTA ? r.E : (int64_t)r.H * r.E; }
        else if (r.kind == MIX_GLA) {
          if (which == 18) { dst = &r.a_up; want = (int64_t)r.rank * r.H * r.D; }
          else if (which == 19) { dst = &r.a_bias; want = (int64_t)r.H * r.D; }
        }
        else if (which == 13) { dst = &r.cv.w; want = (int64_t)r.cv.C * r.cv.taps; }
        else if (which == 14) { dst = &r.cv.b; want = r.cv.C; }
        else if (which == 15) { dst = &r.dt_bias; want = r.H; }
        else if (which == 16) { dst = &r.A_log; want = r.H; }
        else if (which == 17) { dst = &r.Dskip; want = r.H; }
      }
      if (!dst) return set_error(TLB_ERR_ARG, "tlb_stack_set_vector: unknown vector id for this mixer");
    }
  }
  TLB_REQUIRE(n == want, "tlb_stack_set_vector: length does not match the layer");
  float* p = (float*)*dst;
  if (!p) {
    const int rc = d->alloc((void**)&p, (size_t)n * 4, d->owned);
    if (rc) return rc;
  }
  TLB_CUDA(cudaMemcpy(p, v, (size_t)n * 4, cudaMemcpyHostToDevice));
  *dst = p;
  return TLB_OK;
}

int64_t tlb_stack_state_bytes(void* h) {
  StackDecoder* d = as_stack(h);
  return d ? d->state_bytes : 0;
}

}  // extern "C"

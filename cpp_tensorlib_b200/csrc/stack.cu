// Native driver of the layer-stack decoder (tlb_stack_* in include/tlb200.h): weights, sequence state,
// scratch, and the launch sequences of one token and of a prompt pass on the shared sequence surface
// (decoder_base.cuh).
//
// One token, five launches a layer (three without a feed-forward), all f32 between the products:
//   [norm1 + input projections of all mixers] -> [all mixers, finished heads] ->
//   [(grouped norm of an ssd mixer) + output projections + residual add] ->
//   [norm2 + gate|up + gated unit] -> [down + residual add]
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
  int slot[2] = {};              // mixer m: -1 = attention, else index into rec
  int proj_n = 0, act_n = 0;     // widths of the projected and of the finished row
  int ff = 0;
  float limit = 0.f;
  const float *norm1 = nullptr, *norm2 = nullptr;
  Mat in, out, gu, down;
};

}  // namespace

struct StackDecoder : DecoderBase {
  bool bf16 = true;
  float eps = 0.f, embed_scale = 1.f;
  std::vector<StackLayer> layers;
  Mat embed;
  const float* final_norm = nullptr;
  std::vector<void*> owned;
  long long state_bytes = 0;
  int proj_max = 0, act_max = 0, ff_max = 0, conv_max = 0, gate_max = 0, o_max = 0, q_max = 0, chunk = 0;
  // one token
  float *x = nullptr, *proj = nullptr, *act = nullptr, *mb = nullptr;
  // prompt pass: rows of pf_rows tokens (hr, actr and ffr in the product's operand type)
  int pf_rows = 0;
  float *xr = nullptr, *projr = nullptr, *orr = nullptr, *tmpr = nullptr, *gath = nullptr;
  float2 *gater = nullptr, *normr = nullptr;
  void *convr = nullptr, *chunkr = nullptr, *hr = nullptr, *qr = nullptr, *actr = nullptr, *ffr = nullptr, *hg = nullptr;
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
  int product(DeviceCtx* c, const void* a, long long lda, const Mat& w, float* C, long long ldc, bool add, int rows,
              cudaStream_t s);
};

int StackDecoder::ready() const {
  bool ok = embed.W && final_norm;
  for (auto& L : layers) {
    ok = ok && L.norm1 && L.in.W && L.out.W && (!L.ff || (L.norm2 && L.gu.W && L.down.W));
    if (L.has_attn) ok = ok && L.at.qn && L.at.kn;
    for (int i = 0; i < L.n_rec; i++) {
      const RecurP& r = L.rec[i];
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
  auto gemv = [&](const Mat& w, const float* in, float* y, int epi, const float* nw, int n_off, int n_len, int groups,
                  float nscale, float limit) {
    RowGemv g{};
    g.x = in; g.W = w.W; g.N = w.N; g.K = w.K; g.ldw = w.ld;
    g.nw = nw; g.n_off = n_off; g.n_len = n_len; g.n_groups = groups; g.eps = eps; g.nscale = nscale;
    g.y = y; g.epi = epi; g.limit = limit;
    return row_gemv_launch(c, g, bf16, s);
  };
  RUN(embed_scaled_launch(embed.W, d_tok, x, hidden, embed.ld, embed_scale, 1, bf16, s));
  for (auto& L : layers) {
    RUN(gemv(L.in, x, proj, 0, L.norm1, 0, hidden, 1, 1.f, 0.f));
    RUN(mixers_decode_launch(L.has_attn ? &L.at : nullptr, L.rec, L.n_rec, proj, act, d_pos, bf16, s));
    const RecurP* nr = nullptr;   // the grouped norm of an ssd mixer runs in front of the output projection
    int ng = 1;
    for (int i = 0; i < L.n_rec; i++)
      if (L.rec[i].kind == MIX_SSD) { nr = &L.rec[i]; ng = L.norm_groups[i]; }
    RUN(gemv(L.out, act, x, 1, nr ? nr->norm : nullptr, nr ? nr->oa : 0, nr ? nr->H * nr->E : 0, ng,
             nr ? nr->out_scale : 1.f, 0.f));
    if (L.ff) {
      RUN(gemv(L.gu, x, mb, 2, L.norm2, 0, hidden, 1, 1.f, L.limit));
      RUN(gemv(L.down, mb, x, 1, nullptr, 0, 0, 1, 1.f, 0.f));
    }
  }
  RUN(gemv(embed, x, logits, 0, final_norm, 0, hidden, 1, 1.f, 0.f));
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
      const size_t n = bf16 && recur_chunk_eligible(L.rec[i]) ? recur_chunk_scratch_bytes(L.rec[i], rows) : 0;
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

int StackDecoder::prefill_pass(const int* d_ids, int rows, int pos, cudaStream_t s) {
  DeviceCtx* c = nullptr;
  int rc = get_ctx(&c);
  if (rc) return rc;
#define PF(expr) do { rc = (expr); if (rc) return rc; } while (0)
  const int E8 = pad8(hidden);
  PF(embed_scaled_launch(embed.W, d_ids, xr, hidden, embed.ld, embed_scale, rows, bf16, s));
  for (auto& L : layers) {
    PF(rms_rows_launch(xr, hidden, L.norm1, hr, E8, hidden, eps, rows, bf16, s));
    PF(product(c, hr, E8, L.in, projr, L.proj_n, false, rows, s));
    if (L.has_attn) {
      PF(attn_rows_prep_launch(L.at, projr, L.proj_n, rows, pos, qr, bf16, s));
      if (bf16 && attn_window_eligible(L.at))
        PF(attn_window_launch(L.at, qr, projr, L.proj_n, actr, L.act_n, rows, pos, s));
      else
        PF(attn_rows_launch(L.at, qr, projr, L.proj_n, actr, L.act_n, rows, pos, bf16, s));
    }
    for (int i = 0; i < L.n_rec; i++) {
      const RecurP& r = L.rec[i];
      const bool chunks = bf16 && recur_chunk_eligible(r);
      PF(recur_rows_conv_launch(r, projr, L.proj_n, rows, pos, convr, gater, normr, chunks, s));
      if (chunks) PF(recur_chunk_launch(r, convr, gater, normr, chunkr, orr, rows, pos, s));
      else PF(recur_rows_scan_launch(r, (const float*)convr, gater, orr, rows, pos, s));
      PF(recur_rows_finish_launch(r, orr, convr, chunks, projr, L.proj_n, actr, L.act_n, L.norm_groups[i], rows, bf16, s));
    }
    PF(product(c, actr, L.act_n, L.out, xr, hidden, true, rows, s));
    if (!L.ff) continue;
    const int F8 = pad8(L.ff);
    PF(rms_rows_launch(xr, hidden, L.norm2, hr, E8, hidden, eps, rows, bf16, s));
    if (bf16) {
      PF(gemm_bf16_tc_launch(c, hr, E8, L.gu.W, L.gu.ld, nullptr, 0, ffr, F8, rows, L.gu.N, L.gu.K, 2, L.limit, s));
      PF(product(c, ffr, F8, L.down, xr, hidden, true, rows, s));
    } else {
      PF(tlb_gemm_f32((const float*)hr, E8, 0, (const float*)L.gu.W, L.gu.ld, 1, tmpr, rows, L.gu.N, L.gu.K, 1.f, 0.f, s));
      PF(glu_rows_launch(tmpr, (float*)ffr, L.ff, L.limit, rows, s));
      PF(product(c, ffr, L.ff, L.down, xr, hidden, true, rows, s));
    }
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
    g.x = xr + (size_t)rows[0] * hidden; g.W = embed.W; g.N = embed.N; g.K = embed.K; g.ldw = embed.ld;
    g.nw = final_norm; g.n_len = hidden; g.n_groups = 1; g.eps = eps; g.nscale = 1.f; g.y = out;
    return row_gemv_launch(c, g, bf16, s);
  }
  TLB_CUDA(cudaMemcpyAsync(idx, rows, (size_t)n * sizeof(int), cudaMemcpyHostToDevice, s));
  rc = gather_rows_launch(xr, idx, gath, hidden, n, s);
  if (!rc) rc = rms_rows_launch(gath, hidden, final_norm, hg, pad8(hidden), hidden, eps, n, bf16, s);
  if (!rc) rc = product(c, hg, pad8(hidden), embed, out, vocab, false, n, s);
  return rc;
}

static int max_i(int a, int b) { return a > b ? a : b; }

static int build(StackDecoder* d, const tlb_stack_cfg* cfg, const tlb_layer_cfg* ls) {
  DeviceCtx* c = nullptr;
  int rc = get_ctx(&c);
  if (rc) return rc;
  d->hidden = cfg->width; d->vocab = cfg->vocab; d->max_ctx = cfg->max_ctx; d->vocab_total = cfg->vocab;
  d->bf16 = !cfg->f32; d->eps = cfg->eps; d->embed_scale = cfg->embed_scale;
  TLB_REQUIRE(d->hidden > 0 && d->vocab > 0 && d->max_ctx > 0 && cfg->n_layers > 0, "tlb_stack_create: bad sizes");
  const int rows = prefill_chunk_rows(4096);
  d->chunk = rows < d->max_ctx ? rows : d->max_ctx;
  d->layers.resize(cfg->n_layers);
  for (int l = 0; l < cfg->n_layers; l++) {
    const tlb_layer_cfg& lc = ls[l];
    StackLayer& L = d->layers[l];
    TLB_REQUIRE(lc.n_mixers >= 1 && lc.n_mixers <= 2 && lc.ff >= 0, "tlb_stack_create: bad layer");
    L.ff = lc.ff; L.limit = lc.limit;
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
        L.slot[m] = -1;
        AttnP& p = L.at;
        p.H = H; p.G = G; p.D = D; p.E = E; p.Dp = pad8(D); p.Ep = pad8(E);
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
        std::vector<float2> f(max_i(1, p.pairs));
        for (int i = 0; i < p.pairs; i++) {
          const double w = pow((double)k.rot_base, -2.0 * i / k.rot_dims);
          f[i].x = (float)w;
          f[i].y = (float)(w - (double)f[i].x);
        }
        float2* df = nullptr;
        if (!rc) rc = d->alloc((void**)&df, f.size() * sizeof(float2), d->owned);
        if (rc) return rc;
        TLB_CUDA(cudaMemcpy(df, f.data(), f.size() * sizeof(float2), cudaMemcpyHostToDevice));
        p.inv_freq = df;
        d->q_max = max_i(d->q_max, H * p.Dp);
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
          TLB_REQUIRE(L.n_rec == 0 || L.rec[0].kind != MIX_SSD, "tlb_stack_create: one ssd mixer a layer");
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
  if (!rc) rc = d->alloc((void**)&d->x, (size_t)d->hidden * 4, d->owned);
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
  if (which == 4) { m = &d->embed; N = d->vocab; K = d->hidden; }
  else {
    TLB_REQUIRE(layer >= 0 && layer < (int64_t)d->layers.size(), "tlb_stack_set_matrix: layer out of range");
    StackLayer& L = d->layers[layer];
    if (which == 0) { m = &L.in; N = L.proj_n; K = d->hidden; }
    else if (which == 1) { m = &L.out; N = d->hidden; K = L.act_n; }
    else if (which == 2) { m = &L.gu; N = 2 * L.ff; K = d->hidden; }
    else if (which == 3) { m = &L.down; N = d->hidden; K = L.ff; }
    else return set_error(TLB_ERR_ARG, "tlb_stack_set_matrix: unknown matrix id");
  }
  TLB_REQUIRE(rows == N && cols == K, "tlb_stack_set_matrix: shape does not match the layer");
  const size_t es = d->es(), ld = (size_t)(cols + 7) & ~(size_t)7;
  if (!m->W) {
    const int rc = d->alloc(&m->W, (size_t)rows * ld * es, d->owned);
    if (rc) return rc;
  }
  m->N = (int)rows; m->K = (int)cols; m->ld = (long long)ld;
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
      TLB_REQUIRE(mixer >= 0 && mixer < 2 && mixer < L.n_rec + (L.has_attn ? 1 : 0), "tlb_stack_set_vector: no such mixer");
      if (L.slot[mixer] < 0) {
        if (which == 10) { dst = &L.at.qn; want = (int64_t)L.at.H * L.at.D; }
        else if (which == 11) { dst = &L.at.kn; want = (int64_t)L.at.G * L.at.D; }
      } else {
        RecurP& r = L.rec[L.slot[mixer]];
        if (which == 12) { dst = &r.norm; want = r.kind == MIX_SSD ? (int64_t)r.H * r.E : r.E; }
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

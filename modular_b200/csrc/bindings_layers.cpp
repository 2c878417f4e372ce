// Bindings of the layer kernels that exist in bf16 and fp32: the fp32 residual seam, latent attention of any size, the
// gated delta rule, token-id expert routing and the fp32 products.
#include "bindings.h"

#include "common/api.h"

namespace py = pybind11;
using torch::Tensor;
using namespace mb::bind;
typedef c10::optional<Tensor> Opt;

namespace {

int dtype_of(const Tensor& t, const char* what) {
  TORCH_CHECK(t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat, what, ": bf16 or fp32 expected");
  return t.scalar_type() == at::kFloat ? 1 : 0;
}
bool given(const Opt& t) { return t.has_value() && t->defined(); }
// a CUDA matrix with unit column stride of `dtype`; returns its row stride
int ld_of(const Tensor& t, at::ScalarType dtype, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.dim() == 2 && t.stride(1) == 1 && t.scalar_type() == dtype, what,
              ": CUDA matrix of the expected dtype with unit column stride");
  return static_cast<int>(t.stride(0));
}
const int32_t* i32(const Tensor& t, int64_t n, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.scalar_type() == at::kInt && t.numel() >= n, what, ": int32 CUDA tensor");
  return t.data_ptr<int32_t>();
}
const float* f32(const Tensor& t, int64_t n, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.scalar_type() == at::kFloat && t.numel() >= n, what, ": fp32 CUDA tensor");
  return t.data_ptr<float>();
}

void residual_norm(Tensor& x, const Opt& ids, const Opt& table, double scale, const Opt& a, const Opt& b, const Opt& e,
                   const Opt& inverse, int top_k, double pair_w, const Opt& rows, const Opt& w1, const Opt& n1,
                   const Opt& w2, const Opt& n2, const Opt& scatter, int cols, bool store_x, double eps, int n_rows,
                   const Opt& norm_a, const Opt& norm_b, double ab_scale, const Opt& c, double mult, const Opt& inject,
                   double inject_scale, const Opt& step) {
  MbResidualNorm p = {};
  p.ab_scale = static_cast<float>(ab_scale); p.mult = static_cast<float>(mult);
  p.ldx = ld_of(x, at::kFloat, "x");
  p.x = x.data_ptr<float>();
  p.cols = cols; p.cols_pad = static_cast<int>(x.size(1)); p.store_x = store_x; p.eps = static_cast<float>(eps);
  p.n_rows = n_rows;
  const int64_t T = x.size(0);
  at::ScalarType dt = given(w1) ? w1->scalar_type() : given(a) ? a->scalar_type() : at::kBFloat16;
  if (given(table)) {
    TORCH_CHECK(given(ids) && ids->scalar_type() == at::kLong && ids->numel() >= T, "residual_norm: ids");
    p.ld_table = ld_of(*table, dt, "table");
    TORCH_CHECK(table->size(1) == p.cols_pad, "residual_norm: table width");
    p.table = table->data_ptr(); p.ids = ids->data_ptr<int64_t>(); p.scale = static_cast<float>(scale);
    p.vocab = static_cast<int>(table->size(0));
  }
  auto branch = [&](const Opt& t, const char* what, int64_t min_rows) {
    const int ld = ld_of(*t, dt, what);
    TORCH_CHECK(t->size(1) >= p.cols_pad && t->size(0) >= min_rows, "residual_norm: ", what, " shape");
    return ld;
  };
  if (given(a)) { p.lda = branch(a, "a", T); p.a = a->data_ptr(); }
  if (given(b)) { p.ldb = branch(b, "b", T); p.b = b->data_ptr(); }
  auto weight = [&](const Opt& t, const char* what) {
    TORCH_CHECK(t->is_cuda() && t->is_contiguous() && t->scalar_type() == dt && t->numel() >= p.cols_pad, "residual_norm: ", what);
    return t->data_ptr();
  };
  if (given(norm_a)) { TORCH_CHECK(given(a), "residual_norm: norm_a without a"); p.norm_a = weight(norm_a, "norm_a"); }
  if (given(norm_b)) { TORCH_CHECK(given(b), "residual_norm: norm_b without b"); p.norm_b = weight(norm_b, "norm_b"); }
  if (given(c)) { p.ldc = branch(c, "c", T); p.c = c->data_ptr(); }
  if (given(step)) p.step = weight(step, "step");
  if (given(inject)) {
    TORCH_CHECK(given(ids) && ids->scalar_type() == at::kLong && ids->numel() >= T, "residual_norm: ids");
    p.ld_inject = ld_of(*inject, dt, "inject");
    TORCH_CHECK(inject->size(1) == p.cols_pad && (!given(table) || table->size(0) == inject->size(0)), "residual_norm: inject shape");
    p.inject = inject->data_ptr(); p.inject_scale = static_cast<float>(inject_scale);
    p.ids = ids->data_ptr<int64_t>(); p.vocab = static_cast<int>(inject->size(0));
  }
  if (given(e)) {
    p.lde = branch(e, "e", T * top_k); p.e = e->data_ptr();
    TORCH_CHECK(given(inverse), "residual_norm: inverse");
    p.inverse = i32(*inverse, T * top_k, "inverse"); p.top_k = top_k; p.pair_w = static_cast<float>(pair_w);
  }
  if (given(rows)) p.rows = i32(*rows, n_rows, "rows");
  else TORCH_CHECK(n_rows <= T, "residual_norm: rows");
  if (given(w1)) {
    TORCH_CHECK(given(n1) && w1->is_contiguous() && w1->numel() >= p.cols_pad, "residual_norm: w1 / n1");
    p.w1 = w1->data_ptr(); p.ld1 = branch(n1, "n1", n_rows); p.n1 = n1->data_ptr();
  }
  if (given(w2)) {
    TORCH_CHECK(given(n2) && w2->is_contiguous() && w2->scalar_type() == dt && w2->numel() >= p.cols_pad, "residual_norm: w2 / n2");
    p.w2 = w2->data_ptr(); p.n2 = n2->data_ptr();
    if (given(scatter)) {
      TORCH_CHECK(scatter->dim() == 2, "residual_norm: scatter");
      p.k2 = static_cast<int>(scatter->size(1));
      p.scatter = i32(*scatter, T * p.k2, "scatter");
      p.ld2 = branch(n2, "n2", T * p.k2);
    } else {
      p.ld2 = branch(n2, "n2", n_rows);
    }
  }
  check_rc(mb_residual_norm(&p, dt == at::kFloat ? 1 : 0, cur_stream()), "residual_norm");
}

// seam with norms on both sides of a branch, see MbSandwichNorm
void sandwich_norm(Tensor& x, const Opt& ids, const Opt& table, double scale, const Opt& inject_ids, const Opt& inject, const Opt& a,
                   const Opt& e, const Opt& inverse, const Opt& pair_w, const Opt& rows, const Opt& w_u, const Opt& b_u, double mult,
                   const Opt& w1, const Opt& b1, const Opt& n1, int cols, bool store_x, double eps, int n_rows) {
  MbSandwichNorm p = {};
  p.ldx = ld_of(x, at::kFloat, "x"); p.x = x.data_ptr<float>();
  p.cols = cols; p.cols_pad = static_cast<int>(x.size(1)); p.store_x = store_x; p.eps = static_cast<float>(eps); p.n_rows = n_rows;
  p.scale = static_cast<float>(scale); p.mult = static_cast<float>(mult);
  const int64_t T = x.size(0);
  const at::ScalarType dt = given(w1) ? w1->scalar_type() : given(a) ? a->scalar_type() : given(e) ? e->scalar_type() : at::kBFloat16;
  auto matrix = [&](const Opt& t, const char* what, int64_t min_rows) {
    const int ld = ld_of(*t, dt, what);
    TORCH_CHECK(t->size(1) >= p.cols_pad && t->size(0) >= min_rows, "sandwich_norm: ", what, " shape");
    return ld;
  };
  auto index = [&](const Opt& t, const char* what) {
    TORCH_CHECK(given(t) && t->is_cuda() && t->is_contiguous() && t->scalar_type() == at::kLong && t->numel() >= T, "sandwich_norm: ", what);
    return t->data_ptr<int64_t>();
  };
  auto weight = [&](const Opt& t, const char* what) -> const void* {
    if (!given(t)) return nullptr;
    TORCH_CHECK(t->is_cuda() && t->is_contiguous() && t->scalar_type() == dt && t->numel() >= p.cols_pad, "sandwich_norm: ", what);
    return t->data_ptr();
  };
  if (given(table)) {
    p.ld_table = matrix(table, "table", 0); p.table = table->data_ptr(); p.ids = index(ids, "ids"); p.vocab = static_cast<int>(table->size(0));
  }
  if (given(inject)) {
    p.ld_inject = matrix(inject, "inject", 0); p.inject = inject->data_ptr(); p.inject_ids = index(inject_ids, "inject_ids");
    p.inject_rows = static_cast<int>(inject->size(0));
  }
  if (given(a)) { p.lda = matrix(a, "a", T); p.a = a->data_ptr(); }
  if (given(e)) {
    TORCH_CHECK(given(inverse) && inverse->dim() == 2 && given(pair_w), "sandwich_norm: inverse [T, k] and pair_w");
    p.top_k = static_cast<int>(inverse->size(1));
    p.lde = matrix(e, "e", T * p.top_k); p.e = e->data_ptr();
    p.inverse = i32(*inverse, T * p.top_k, "inverse"); p.pair_w = f32(*pair_w, T * p.top_k, "pair_w");
  }
  if (given(rows)) p.rows = i32(*rows, n_rows, "rows");
  else TORCH_CHECK(n_rows <= T, "sandwich_norm: rows");
  p.w_u = weight(w_u, "w_u"); p.b_u = weight(b_u, "b_u"); p.w1 = weight(w1, "w1"); p.b1 = weight(b1, "b1");
  if (given(w1)) { TORCH_CHECK(given(n1), "sandwich_norm: n1"); p.ld1 = matrix(n1, "n1", n_rows); p.n1 = n1->data_ptr(); }
  check_rc(mb_sandwich_norm(&p, dt == at::kFloat ? 1 : 0, cur_stream()), "sandwich_norm");
}

// seam with elementwise norms and an optional token shift, see MbTanhSeam; `x_out` may be `x` where there is no shift
void tanh_seam(const Opt& x, const Opt& x_out, const Opt& ids, const Opt& table, double scale, const Opt& a, const Opt& e,
               const Opt& inverse, const Opt& pair_w, const Opt& self, const Opt& rows, const Opt& w_u, const Opt& b_u, double alpha_u,
               const Opt& w1, const Opt& b1, double alpha_1, const Opt& n1, const Opt& shift, const Opt& prev, const Opt& state_idx,
               const Opt& q_start, const Opt& q_len, const Opt& kv_len, bool one_token, int cols_pad, int n_rows) {
  MbTanhSeam p = {};
  p.cols_pad = cols_pad; p.n_rows = n_rows; p.scale = static_cast<float>(scale);
  p.alpha_u = static_cast<float>(alpha_u); p.alpha_1 = static_cast<float>(alpha_1);
  const at::ScalarType dt = given(w1) ? w1->scalar_type() : given(w_u) ? w_u->scalar_type() : given(table) ? table->scalar_type() : at::kBFloat16;
  int64_t T = n_rows;
  auto stream_rows = [&](const Opt& t, const char* what) {
    const int ld = ld_of(*t, at::kFloat, what);
    TORCH_CHECK(t->size(1) >= cols_pad && (p.ldx == 0 || ld == p.ldx), "tanh_seam: ", what, " shape");
    p.ldx = ld;
    T = t->size(0);
    return t->data_ptr<float>();
  };
  TORCH_CHECK(given(x) || given(table), "tanh_seam: x or table");
  if (given(x)) p.x = stream_rows(x, "x");
  if (given(x_out)) {
    const int64_t before = T;
    p.x_out = stream_rows(x_out, "x_out");
    TORCH_CHECK(!given(x) || T == before, "tanh_seam: x_out rows");
  }
  auto matrix = [&](const Opt& t, const char* what, int64_t min_rows) {
    const int ld = ld_of(*t, dt, what);
    TORCH_CHECK(t->size(1) >= cols_pad && t->size(0) >= min_rows, "tanh_seam: ", what, " shape");
    return ld;
  };
  auto weight = [&](const Opt& t, const char* what) -> const void* {
    if (!given(t)) return nullptr;
    TORCH_CHECK(t->is_cuda() && t->is_contiguous() && t->scalar_type() == dt && t->numel() >= cols_pad, "tanh_seam: ", what);
    return t->data_ptr();
  };
  if (given(table)) {
    TORCH_CHECK(given(ids) && ids->is_cuda() && ids->is_contiguous() && ids->scalar_type() == at::kLong && ids->numel() >= T, "tanh_seam: ids");
    p.ld_table = matrix(table, "table", 0); p.table = table->data_ptr(); p.ids = ids->data_ptr<int64_t>();
    p.vocab = static_cast<int>(table->size(0));
  }
  if (given(a)) { p.lda = matrix(a, "a", T); p.a = a->data_ptr(); }
  if (given(e)) {
    TORCH_CHECK(given(inverse) && inverse->dim() == 2 && given(pair_w), "tanh_seam: inverse [T, k] and pair_w");
    p.top_k = static_cast<int>(inverse->size(1));
    p.lde = matrix(e, "e", T * p.top_k); p.e = e->data_ptr();
    p.inverse = i32(*inverse, T * p.top_k, "inverse"); p.pair_w = f32(*pair_w, T * p.top_k, "pair_w");
    if (given(self)) { p.ld_self = matrix(self, "self", T); p.self = self->data_ptr(); }
  }
  if (given(rows)) p.rows = i32(*rows, n_rows, "rows");
  else TORCH_CHECK(n_rows <= T, "tanh_seam: rows");
  p.w_u = weight(w_u, "w_u"); p.b_u = weight(b_u, "b_u"); p.w1 = weight(w1, "w1"); p.b1 = weight(b1, "b1");
  if (given(w1)) { TORCH_CHECK(given(n1), "tanh_seam: n1"); p.ld1 = matrix(n1, "n1", n_rows); p.n1 = n1->data_ptr(); }
  if (given(shift)) {
    TORCH_CHECK(given(prev) && prev->is_cuda() && prev->is_contiguous() && prev->scalar_type() == at::kFloat && prev->dim() == 2 &&
                    prev->size(1) == cols_pad && given(state_idx) && given(q_start) && given(q_len) && given(kv_len), "tanh_seam: shift state");
    p.shift = weight(shift, "shift"); p.prev = prev->data_ptr<float>();
    p.B = q_len->numel(); p.one_token = one_token;
    p.state_idx = i32(*state_idx, p.B, "state_idx"); p.q_start = i32(*q_start, p.B, "q_start");
    p.q_len = i32(*q_len, p.B, "q_len"); p.kv_len = i32(*kv_len, p.B, "kv_len");
  }
  check_rc(mb_tanh_seam(&p, dt == at::kFloat ? 1 : 0, cur_stream()), "tanh_seam");
}

// window, sink and output gate of an attention call; `use` is what the C interface takes (null: none of them)
struct AttnOptions {
  MbAttnOptions o = {};
  const MbAttnOptions* use = nullptr;
  AttnOptions(int window, const Opt& sink, const Opt& gate, double gate_mult, int64_t T, int64_t heads, at::ScalarType dt, const char* what) {
    o.window = window;
    o.gate_mult = static_cast<float>(gate_mult);
    if (given(sink)) o.sink = f32(*sink, heads, "sink");
    if (given(gate)) {
      o.ld_gate = ld_of(*gate, dt, "gate"); o.gate = gate->data_ptr();
      TORCH_CHECK(gate->size(0) >= T && gate->size(1) >= heads, what, ": gate [T, heads]");
    }
    if (window > 0 || o.sink || o.gate) use = &o;
  }
};

void latent_post_down(const Tensor& x, int q_rank, const Opt& gamma_q, const Opt& q_out, int kv_off, int R, int Rp,
                      const Opt& gamma_kv, int rot_dim, int Dp, int dims, bool interleaved, double eps,
                      const Tensor& positions, const Tensor& cos_sin, const Tensor& slots, const Opt& cache) {
  const int dt = dtype_of(x, "x"), ld = ld_of(x, x.scalar_type(), "x");
  const int64_t T = x.size(0);
  TORCH_CHECK(slots.scalar_type() == at::kLong && slots.numel() >= T && cos_sin.dim() == 2 && cos_sin.size(1) == dims &&
                  q_rank <= x.size(1) && kv_off + (kv_off >= 0 ? R + rot_dim : 0) <= x.size(1),
              "latent_post_down: slots / cos_sin / columns");
  int ld_q = 0, q_pad = 0;
  if (q_rank > 0) {
    TORCH_CHECK(given(gamma_q) && given(q_out) && gamma_q->numel() >= q_rank && gamma_q->scalar_type() == x.scalar_type() &&
                    q_out->size(0) >= T, "latent_post_down: query latent");
    ld_q = ld_of(*q_out, x.scalar_type(), "q_out"); q_pad = static_cast<int>(q_out->size(1));
  }
  int page = 1, ld_cache = 0;
  int64_t page_stride = 0;
  if (kv_off >= 0) {
    TORCH_CHECK(given(gamma_kv) && gamma_kv->numel() >= R && gamma_kv->scalar_type() == x.scalar_type() && given(cache) &&
                    cache->dim() == 3 && cache->stride(2) == 1 && cache->size(2) >= Rp + Dp && cache->scalar_type() == x.scalar_type(),
                "latent_post_down: cache");
    page = static_cast<int>(cache->size(1)); ld_cache = static_cast<int>(cache->stride(1)); page_stride = cache->stride(0);
  }
  check_rc(mb_latent_post_down(x.data_ptr(), ld, static_cast<int>(T), q_rank, q_pad, optptr(gamma_q),
                               const_cast<void*>(optptr(q_out)), ld_q, kv_off, R, Rp, optptr(gamma_kv), rot_dim, Dp, dims,
                               interleaved ? 1 : 0, static_cast<float>(eps), i32(positions, T, "positions"),
                               f32(cos_sin, 0, "cos_sin"), slots.data_ptr<int64_t>(), const_cast<void*>(optptr(cache)), page,
                               page_stride, ld_cache, dt, cur_stream()),
           "latent_post_down");
}

// q_lat [T, h, Rp], q_rope [T, h, Dp] (any token stride, heads contiguous blocks), cache [pages, page, >= Rp + Dp]
void latent_attention(const Tensor& q_lat, const Tensor& q_rope, const Tensor& cache, const Tensor& block_table,
                      const Tensor& q_start, const Tensor& q_len, const Tensor& kv_len, Tensor& out, double scale,
                      const Opt& sink, bool one_token, const Opt& ws, bool allow_tc, int window, const Opt& gate, double gate_mult) {
  const int dt = dtype_of(q_lat, "q_lat");
  TORCH_CHECK(q_lat.is_cuda() && q_lat.dim() == 3 && q_lat.stride(2) == 1 && q_rope.dim() == 3 && q_rope.stride(2) == 1 &&
                  out.is_contiguous() && out.sizes() == q_lat.sizes() && q_rope.size(0) == q_lat.size(0) &&
                  q_rope.size(1) == q_lat.size(1) && q_rope.scalar_type() == q_lat.scalar_type() &&
                  out.scalar_type() == q_lat.scalar_type() && cache.scalar_type() == q_lat.scalar_type() && cache.dim() == 3 &&
                  cache.stride(2) == 1 && cache.size(2) >= q_lat.size(2) + q_rope.size(2) && block_table.stride(1) == 1 &&
                  block_table.scalar_type() == at::kInt,
              "latent_attention layout");
  const int T = q_lat.size(0), h = q_lat.size(1), R = q_lat.size(2), D = q_rope.size(2), B = q_len.numel();
  const AttnOptions opt(window, sink, gate, gate_mult, T, h, q_lat.scalar_type(), "latent_attention");
  const int32_t *qs = i32(q_start, B, "q_start"), *ql = i32(q_len, B, "q_len"), *kl = i32(kv_len, B, "kv_len");
  const int32_t* bt = block_table.data_ptr<int32_t>();
  const int page = cache.size(1), bts = block_table.stride(0), ldc = cache.stride(1);
  TORCH_CHECK(block_table.size(0) >= B, "latent_attention: block table rows");
  const bool mma = dt == 0 && D == 64 && (R == 64 || R == 128 || R == 192 || R == 256 || R == 384 || R == 512) &&
                   q_lat.stride(1) == R;
  // 512-wide latents with a multiple of 128 heads: tcgen05 kernel, which addresses contiguous query rows
  if (mma && allow_tc && q_lat.is_contiguous() && q_rope.stride(0) == h * q_rope.stride(1) && ldc == R + D && cache.stride(0) % (R + D) == 0 &&
      mb_mla_tc_usable(T, T, h, R, page)) {
    if (one_token) {
      check_rc(mb_mla_decode_tc(q_lat.data_ptr(), q_rope.data_ptr(), out.data_ptr(), cache.data_ptr(), cache.stride(0),
                                cache.size(0), bt, bts, qs, ql, kl, T, B, h, page, scale, opt.use,
                                static_cast<int>(q_rope.stride(1)), error_flag(), cur_stream()),
               "mla_decode_tc");
    } else {
      auto scratch = at::empty({2 * static_cast<int64_t>(T)}, q_start.options());
      check_rc(mb_mla_prefill_tc(q_lat.data_ptr(), q_rope.data_ptr(), out.data_ptr(), cache.data_ptr(), cache.stride(0),
                                 cache.size(0), bt, bts, qs, ql, kl, T, B, h, page, scale, opt.use,
                                 static_cast<int>(q_rope.stride(1)), scratch.data_ptr<int32_t>(),
                                 error_flag(), cur_stream()),
               "mla_prefill_tc");
    }
    return;
  }
  if (mma) {
    check_rc(mb_mla_paged_attention_ex(q_lat.data_ptr(), q_lat.stride(0), q_rope.data_ptr(), q_rope.stride(0), q_rope.stride(1),
                                       out.data_ptr(), cache.data_ptr(), cache.stride(0), ldc, bt, bts, qs, ql, kl, T, B, h, R, page, scale, opt.use,
                                       given(ws) ? ws->data_ptr() : nullptr, given(ws) ? ws->nbytes() : 0, num_sms(),
                                       cur_stream()),
             "mla_paged_attention");
    return;
  }
  check_rc(mb_latent_attention(q_lat.data_ptr(), q_lat.stride(0), q_lat.stride(1), q_rope.data_ptr(), q_rope.stride(0),
                               q_rope.stride(1), out.data_ptr(), out.stride(0), out.stride(1), cache.data_ptr(),
                               cache.stride(0), ldc, page, bt, bts, qs, ql, kl, T, B, h, R, D, scale, opt.use, dt, cur_stream()),
           "latent_attention");
}

// x: projection rows with the column blocks of q, k, v and beta at the given offsets; see MbDelta for the rest
void delta_rule(const Tensor& x, int q_off, int k_off, int v_off, int b_off, const Tensor& conv_w, const Opt& z,
                const Tensor& A_log, const Tensor& dt_bias, const Tensor& gate, const Tensor& norm_w, double eps,
                std::vector<Tensor>& scratch, Tensor& out, Tensor& state, Tensor& conv_state, const Tensor& state_idx,
                const Tensor& q_start, const Tensor& q_len, const Tensor& kv_len, int heads, int kv_heads, int dim, int vdim,
                bool one_token, int a_off, bool gate_silu, double out_mult) {
  MbDelta p = {};
  const int dt = dtype_of(x, "x");
  const at::ScalarType st = x.scalar_type();
  p.T = x.size(0); p.B = q_len.numel();
  p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim; p.one_token = one_token;
  p.dim_pad = mb_delta_dim_pad(dim);
  TORCH_CHECK(p.dim_pad > 0, "delta_rule: key width ", dim, " is beyond the supported maximum");
  const int64_t T = p.T, C = 2ll * kv_heads * dim + static_cast<int64_t>(heads) * vdim;
  p.x = x.data_ptr(); p.ldx = ld_of(x, st, "x");
  p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.b_off = b_off;
  TORCH_CHECK(q_off + kv_heads * dim <= x.size(1) && k_off + kv_heads * dim <= x.size(1) &&
                  v_off + heads * vdim <= x.size(1) && b_off + heads <= x.size(1), "delta_rule: columns");
  TORCH_CHECK(conv_w.is_contiguous() && conv_w.scalar_type() == st && conv_w.dim() == 2 && conv_w.size(0) == C, "delta_rule: conv_w");
  p.conv_w = conv_w.data_ptr(); p.taps = conv_w.size(1);
  if (given(z)) {
    p.ldz = ld_of(*z, at::kFloat, "z"); p.z = z->data_ptr<float>();
    TORCH_CHECK(z->size(0) >= T && z->size(1) >= heads * dim, "delta_rule: z");
  } else {                                       // one decay per head, from columns of x
    TORCH_CHECK(a_off >= 0 && a_off + heads <= x.size(1), "delta_rule: a_off");
    p.a_off = a_off;
  }
  p.gate_silu = gate_silu; p.out_mult = static_cast<float>(out_mult);
  p.A_log = f32(A_log, heads, "A_log"); p.dt_bias = f32(dt_bias, static_cast<int64_t>(heads) * (given(z) ? dim : 1), "dt_bias");
  p.ld_gate = ld_of(gate, st, "gate"); p.gate = gate.data_ptr();
  TORCH_CHECK(gate.size(0) >= T && gate.size(1) >= heads * vdim, "delta_rule: gate");
  TORCH_CHECK(norm_w.is_contiguous() && norm_w.scalar_type() == st && norm_w.numel() >= vdim, "delta_rule: norm_w");
  p.norm_w = norm_w.data_ptr(); p.eps = static_cast<float>(eps);
  TORCH_CHECK(scratch.size() == 7, "delta_rule: scratch is {q, k, g, v, beta, kq, o}");
  const int64_t need[7] = {T * kv_heads * p.dim_pad, T * kv_heads * p.dim_pad, T * heads * (given(z) ? p.dim_pad : 1), T * heads * vdim,
                           T * heads, T * kv_heads, T * heads * vdim};
  float** dst[7] = {&p.q, &p.k, &p.g, &p.v, &p.beta, &p.kq, &p.o};
  for (int i = 0; i < 7; ++i) *dst[i] = const_cast<float*>(f32(scratch[i], need[i], "delta_rule scratch"));
  p.ld_out = ld_of(out, st, "out"); p.out = out.data_ptr();
  TORCH_CHECK(out.size(0) >= T && out.size(1) >= heads * vdim, "delta_rule: out");
  TORCH_CHECK(state.is_contiguous() && state.scalar_type() == at::kFloat && state.dim() == 4 && state.size(1) == heads &&
                  state.size(2) == vdim && state.size(3) == p.dim_pad, "delta_rule: state [slots, heads, vdim, dim_pad]");
  TORCH_CHECK(conv_state.is_contiguous() && conv_state.scalar_type() == at::kFloat && conv_state.dim() == 3 &&
                  conv_state.size(1) == C && conv_state.size(2) == p.taps - 1, "delta_rule: conv_state [slots, channels, taps - 1]");
  p.state = state.data_ptr<float>(); p.conv_state = conv_state.data_ptr<float>();
  p.state_idx = i32(state_idx, p.B, "state_idx"); p.q_start = i32(q_start, p.B, "q_start");
  p.q_len = i32(q_len, p.B, "q_len"); p.kv_len = i32(kv_len, p.B, "kv_len");
  check_rc(mb_delta_rule(&p, dt, num_sms(), cur_stream()), "delta_rule");
}

// x: projection rows with the column blocks of q, k and v at the given offsets; see MbGla
void gla(const Tensor& x, int q_off, int k_off, int v_off, const Tensor& z, const Tensor& z_bias, double q_scale, double inv_tau,
         const Tensor& gate, bool gate_silu, double out_mult, const Tensor& norm_w, double eps, int norm_dim, Tensor& o, Tensor& out,
         Tensor& state, const Tensor& state_idx, const Tensor& q_start, const Tensor& q_len, const Tensor& kv_len, int heads, int dim,
         int vdim, bool one_token, bool allow_chunks) {
  MbGla p = {};
  const at::ScalarType st = x.scalar_type();
  p.T = x.size(0); p.B = q_len.numel(); p.heads = heads; p.dim = dim; p.vdim = vdim; p.one_token = one_token;
  p.dim_pad = mb_delta_dim_pad(dim);
  TORCH_CHECK(p.dim_pad > 0, "gla: key width ", dim, " is beyond the supported maximum");
  const int64_t T = p.T;
  p.x = x.data_ptr(); p.ldx = ld_of(x, st, "x"); p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
  TORCH_CHECK(q_off + heads * dim <= x.size(1) && k_off + heads * dim <= x.size(1) && v_off + heads * vdim <= x.size(1), "gla: columns");
  p.ldz = ld_of(z, at::kFloat, "z"); p.z = z.data_ptr<float>();
  TORCH_CHECK(z.size(0) >= T && z.size(1) >= heads * dim, "gla: z");
  p.z_bias = f32(z_bias, static_cast<int64_t>(heads) * dim, "z_bias");
  p.q_scale = static_cast<float>(q_scale); p.inv_tau = static_cast<float>(inv_tau);
  p.ld_gate = ld_of(gate, st, "gate"); p.gate = gate.data_ptr(); p.gate_silu = gate_silu; p.out_mult = static_cast<float>(out_mult);
  TORCH_CHECK(gate.size(0) >= T && gate.size(1) >= heads * vdim, "gla: gate");
  TORCH_CHECK(norm_w.is_contiguous() && norm_w.scalar_type() == st && norm_w.numel() >= vdim, "gla: norm_w");
  p.norm_w = norm_w.data_ptr(); p.eps = static_cast<float>(eps); p.norm_dim = norm_dim;
  p.o = const_cast<float*>(f32(o, one_token ? 0 : T * heads * vdim, "gla: o"));
  p.ld_out = ld_of(out, st, "out"); p.out = out.data_ptr();
  TORCH_CHECK(out.size(0) >= T && out.size(1) >= heads * vdim, "gla: out");
  TORCH_CHECK(state.is_contiguous() && state.scalar_type() == at::kFloat && state.dim() == 4 && state.size(1) == heads &&
                  state.size(2) == vdim && state.size(3) == p.dim_pad, "gla: state [slots, heads, vdim, dim_pad]");
  p.state = state.data_ptr<float>();
  p.state_idx = i32(state_idx, p.B, "state_idx"); p.q_start = i32(q_start, p.B, "q_start");
  p.q_len = i32(q_len, p.B, "q_len"); p.kv_len = i32(kv_len, p.B, "kv_len");
  const int dt = dtype_of(x, "x"), chunks = allow_chunks ? mb_gla_chunks(&p, dt) : 0;
  Tensor plan, qk, ends;
  if (chunks > 0) {
    plan = at::empty({2, chunks}, q_start.options());
    qk = at::empty({chunks, heads, 4, 64, p.dim_pad}, x.options());
    ends = at::empty({chunks, heads, p.dim_pad}, z.options());
    int32_t* t = plan.data_ptr<int32_t>();
    check_rc(mb_attention_plan(p.q_len, p.B, 64, chunks, t, t + chunks, cur_stream()), "gla plan");
    p.tile_seq = t; p.tile_q0 = t + chunks; p.n_tiles = chunks; p.qk = qk.data_ptr(); p.ends = ends.data_ptr<float>();
  }
  check_rc(mb_gla(&p, dt, num_sms(), cur_stream()), "gla");
}

// x: projection rows with the column blocks of r, k, v and the removal rates at the given offsets; see MbGeneralDelta
void general_delta(const Tensor& x, int r_off, int k_off, int v_off, int a_off, const Tensor& a_bias, const Tensor& z, const Tensor& z_bias,
                   const Tensor& gate, const Tensor& norm_w, double eps, int norm_dim, Tensor& rows, Tensor& o, Tensor& out, Tensor& state,
                   const Tensor& state_idx, const Tensor& q_start, const Tensor& q_len, const Tensor& kv_len, int heads, int dim, int vdim,
                   bool one_token) {
  MbGeneralDelta p = {};
  const at::ScalarType st = x.scalar_type();
  p.T = x.size(0); p.B = q_len.numel(); p.heads = heads; p.dim = dim; p.vdim = vdim; p.one_token = one_token;
  p.dim_pad = mb_delta_dim_pad(dim);
  TORCH_CHECK(p.dim_pad > 0, "general_delta: key width ", dim, " is beyond the supported maximum");
  const int64_t T = p.T, HD = static_cast<int64_t>(heads) * dim, HV = static_cast<int64_t>(heads) * vdim;
  p.x = x.data_ptr(); p.ldx = ld_of(x, st, "x"); p.r_off = r_off; p.k_off = k_off; p.v_off = v_off; p.a_off = a_off;
  TORCH_CHECK(r_off + HD <= x.size(1) && k_off + HD <= x.size(1) && v_off + HV <= x.size(1) && a_off + HD <= x.size(1),
              "general_delta: columns");
  p.a_bias = f32(a_bias, HD, "a_bias"); p.z_bias = f32(z_bias, HD, "z_bias");
  p.ldz = ld_of(z, at::kFloat, "z"); p.z = z.data_ptr<float>();
  TORCH_CHECK(z.size(0) >= T && z.size(1) >= HD, "general_delta: z");
  p.ld_gate = ld_of(gate, st, "gate"); p.gate = gate.data_ptr();
  TORCH_CHECK(gate.size(0) >= T && gate.size(1) >= HV, "general_delta: gate");
  TORCH_CHECK(norm_w.is_cuda() && norm_w.is_contiguous() && norm_w.scalar_type() == st && norm_w.numel() >= HV, "general_delta: norm_w");
  p.norm_w = norm_w.data_ptr(); p.eps = static_cast<float>(eps); p.norm_dim = norm_dim;
  const bool fused = one_token && vdim <= (p.dim_pad <= 256 ? 128 : 64);       // no scratch where one launch does it all
  p.rows = const_cast<float*>(f32(rows, fused ? 0 : T * heads * (4 * p.dim_pad + 4), "general_delta: rows"));
  p.o = const_cast<float*>(f32(o, fused ? 0 : T * HV, "general_delta: o"));
  p.ld_out = ld_of(out, st, "out"); p.out = out.data_ptr();
  TORCH_CHECK(out.size(0) >= T && out.size(1) >= HV, "general_delta: out");
  TORCH_CHECK(state.is_contiguous() && state.scalar_type() == at::kFloat && state.dim() == 4 && state.size(1) == heads &&
                  state.size(2) == vdim && state.size(3) == p.dim_pad, "general_delta: state [slots, heads, vdim, dim_pad]");
  p.state = state.data_ptr<float>();
  p.state_idx = i32(state_idx, p.B, "state_idx"); p.q_start = i32(q_start, p.B, "q_start");
  p.q_len = i32(q_len, p.B, "q_len"); p.kv_len = i32(kv_len, p.B, "kv_len");
  check_rc(mb_general_delta(&p, dtype_of(x, "x"), num_sms(), cur_stream()), "general_delta");
}

// the cache [pages, 2, planes, kv heads, page, head width] at one plane
struct CacheView {
  char *k, *v;
  long long page_stride, head_stride;
  int page, hd;
  CacheView(const Tensor& kv, int plane, int n_kv, const char* what) {
    TORCH_CHECK(kv.is_cuda() && kv.dim() == 6 && kv.is_contiguous() && kv.size(1) == 2 && plane >= 0 && plane < kv.size(2) &&
                    n_kv <= kv.size(3), what, ": cache [pages, 2, planes, kv heads, page, head width]");
    k = static_cast<char*>(kv.data_ptr()) + plane * kv.stride(2) * kv.element_size();
    v = k + kv.stride(1) * kv.element_size();
    page_stride = kv.stride(0); head_stride = kv.stride(3); page = kv.size(4); hd = kv.size(5);
  }
};

// x: projection rows; queries at column 0 .., see MbBlockPrep
void block_prep(Tensor& x, int q_off, int heads, int k_off, int v_off, int kv_heads, int dims, const Tensor& positions,
                const Opt& cos_sin, const Tensor& slots, Tensor& kv, int plane, int silu_off, int silu_n, int relu2_off, int relu2_n,
                const Opt& q_norm, const Opt& k_norm, int norm_dim, double eps, bool halves, const Opt& bias) {
  MbBlockPrep p = {};
  p.x = x.data_ptr(); p.ldx = ld_of(x, x.scalar_type(), "x"); p.T = x.size(0);
  const CacheView c(kv, plane, kv_heads, "block_prep");
  TORCH_CHECK(kv.scalar_type() == x.scalar_type(), "block_prep: cache dtype");
  p.q_off = q_off; p.heads = heads; p.k_off = k_off; p.v_off = v_off; p.kv_heads = kv_heads; p.hd = c.hd; p.dims = dims;
  const int64_t W = x.size(1);
  TORCH_CHECK(q_off + static_cast<int64_t>(heads) * c.hd <= W && k_off + static_cast<int64_t>(kv_heads) * c.hd <= W &&
                  v_off + static_cast<int64_t>(kv_heads) * c.hd <= W && silu_off + silu_n <= W && relu2_off + relu2_n <= W,
              "block_prep: columns out of range");
  if (dims > 0) {
    TORCH_CHECK(given(cos_sin) && cos_sin->dim() == 2 && cos_sin->size(1) == dims, "block_prep: cos_sin");
    p.cos_sin = f32(*cos_sin, 0, "cos_sin");
  }
  TORCH_CHECK(slots.is_cuda() && slots.scalar_type() == at::kLong && slots.numel() >= p.T, "block_prep: slots");
  p.positions = i32(positions, p.T, "positions"); p.slots = slots.data_ptr<int64_t>();
  p.k_cache = c.k; p.v_cache = c.v; p.page_size = c.page; p.page_stride = c.page_stride; p.head_stride = c.head_stride;
  p.silu_off = silu_off; p.silu_n = silu_n; p.relu2_off = relu2_off; p.relu2_n = relu2_n;
  auto weight = [&](const Opt& t) -> const void* {
    if (!given(t)) return nullptr;
    TORCH_CHECK(t->is_cuda() && t->is_contiguous() && t->scalar_type() == x.scalar_type() && t->numel() >= c.hd, "block_prep: norm weight");
    return t->data_ptr();
  };
  p.q_norm = weight(q_norm); p.k_norm = weight(k_norm); p.norm_dim = norm_dim > 0 ? norm_dim : c.hd; p.eps = static_cast<float>(eps);
  p.halves = halves;
  if (given(bias)) p.bias = f32(*bias, std::max<int64_t>(q_off + static_cast<int64_t>(heads) * c.hd,
                                                        std::max(k_off, v_off) + static_cast<int64_t>(kv_heads) * c.hd), "bias");
  check_rc(mb_block_prep(&p, dtype_of(x, "x"), cur_stream()), "block_prep");
}

// q [T, n_q * head width] (row stride free). Tensor cores: `decode_seq` (one row per sequence) or `tile_seq` / `tile_q0`;
// none of them given: the kernel on the CUDA cores.
void window_attention(const Tensor& q, Tensor& out, const Tensor& kv, int plane, const Tensor& block_table, const Tensor& q_start,
                      const Tensor& q_len, const Tensor& kv_len, const Opt& tile_seq, const Opt& tile_q0, const Opt& decode_seq,
                      int n_q, int n_kv, double scale, int window, const Opt& sink, const Opt& gate, double gate_mult) {
  const CacheView c(kv, plane, n_kv, "window_attention");
  const int dt = dtype_of(q, "q"), ldq = ld_of(q, q.scalar_type(), "q"), ldo = ld_of(out, q.scalar_type(), "out");
  const int B = q_len.numel(), T = q.size(0);
  TORCH_CHECK(kv.scalar_type() == q.scalar_type() && q.size(1) >= static_cast<int64_t>(n_q) * c.hd && out.size(0) >= T &&
                  out.size(1) >= static_cast<int64_t>(n_q) * c.hd && block_table.scalar_type() == at::kInt &&
                  block_table.dim() == 2 && block_table.stride(1) == 1 && block_table.size(0) >= B, "window_attention layout");
  const AttnOptions opt(window, sink, gate, gate_mult, T, n_q, q.scalar_type(), "window_attention");
  const int32_t *qs = i32(q_start, B, "q_start"), *ql = i32(q_len, B, "q_len"), *kl = i32(kv_len, B, "kv_len");
  const int32_t* bt = block_table.data_ptr<int32_t>();
  const int bts = block_table.stride(0);
  if (!given(tile_seq) && !given(decode_seq)) {
    check_rc(mb_window_attention(q.data_ptr(), ldq, out.data_ptr(), ldo, c.k, c.v, c.page_stride, c.head_stride, c.page, bt, bts, qs,
                                 ql, kl, T, B, n_q, n_kv, c.hd, static_cast<float>(scale), opt.use, dt, cur_stream()),
             "window_attention");
    return;
  }
  TORCH_CHECK(dt == 0, "window_attention: the tensor-core kernels take bf16");
  const int n_tiles = given(tile_seq) ? tile_seq->numel() : 0, n_dec = given(decode_seq) ? decode_seq->numel() : 0;
  const long long hd = c.hd, rows_k = plane * kv.stride(2) / hd;
  check_rc(mb_paged_attention_window(q.data_ptr(), ldq, out.data_ptr(), ldo, kv.data_ptr(), kv.numel() / hd, rows_k,
                                     rows_k + kv.stride(1) / hd, kv.stride(0) / hd, bt, bts, qs, ql, kl,
                                     n_tiles ? i32(*tile_seq, n_tiles, "tile_seq") : nullptr,
                                     n_tiles ? i32(*tile_q0, n_tiles, "tile_q0") : nullptr, n_tiles, n_dec,
                                     n_dec ? i32(*decode_seq, n_dec, "decode_seq") : nullptr, n_q, n_kv, c.hd, c.page,
                                     static_cast<float>(scale), opt.use, error_flag(), cur_stream()),
           "paged_attention_window");
}

// x: activated projection rows with the column blocks of q, k and v at the given offsets
void lightning(const Tensor& x, int q_off, int k_off, int v_off, const Tensor& decay, const Tensor& decay_pow, Tensor& o,
               Tensor& state, const Tensor& state_idx, const Tensor& q_start, const Tensor& q_len, const Tensor& kv_len, int heads,
               int dim, int vdim, bool one_token) {
  MbLightning p = {};
  p.T = x.size(0); p.B = q_len.numel(); p.heads = heads; p.dim = dim; p.vdim = vdim; p.one_token = one_token;
  p.dim_pad = mb_delta_dim_pad(dim);
  TORCH_CHECK(p.dim_pad > 0, "lightning: key width ", dim, " is beyond the supported maximum");
  p.x = x.data_ptr(); p.ldx = ld_of(x, x.scalar_type(), "x"); p.q_off = q_off; p.k_off = k_off; p.v_off = v_off;
  TORCH_CHECK(q_off + heads * dim <= x.size(1) && k_off + heads * dim <= x.size(1) && v_off + heads * vdim <= x.size(1),
              "lightning: columns");
  p.decay = f32(decay, heads, "decay"); p.decay_pow = f32(decay_pow, 65ll * heads, "decay_pow");
  p.o = o.data_ptr(); p.ldo = ld_of(o, x.scalar_type(), "o");
  TORCH_CHECK(o.size(0) >= p.T && o.size(1) >= heads * vdim, "lightning: o");
  TORCH_CHECK(state.is_contiguous() && state.scalar_type() == at::kFloat && state.dim() == 4 && state.size(1) == heads &&
                  state.size(2) == vdim && state.size(3) == p.dim_pad, "lightning: state [slots, heads, vdim, dim_pad]");
  p.state = state.data_ptr<float>();
  p.state_idx = i32(state_idx, p.B, "state_idx"); p.q_start = i32(q_start, p.B, "q_start");
  p.q_len = i32(q_len, p.B, "q_len"); p.kv_len = i32(kv_len, p.B, "kv_len");
  check_rc(mb_lightning(&p, dtype_of(x, "x"), num_sms(), cur_stream()), "lightning");
}

}  // namespace

void mb::bind_layers(py::module_& m) {
  const auto none = py::none();
  m.def("residual_norm", &residual_norm, py::arg("x"), py::arg("ids") = none, py::arg("table") = none, py::arg("scale") = 1.0,
        py::arg("a") = none, py::arg("b") = none, py::arg("e") = none, py::arg("inverse") = none, py::arg("top_k") = 0,
        py::arg("pair_w") = 1.0, py::arg("rows") = none, py::arg("w1") = none, py::arg("n1") = none, py::arg("w2") = none,
        py::arg("n2") = none, py::arg("scatter") = none, py::arg("cols") = 0, py::arg("store_x") = true, py::arg("eps") = 1e-6,
        py::arg("n_rows") = 0, py::arg("norm_a") = none, py::arg("norm_b") = none, py::arg("ab_scale") = 1.0, py::arg("c") = none,
        py::arg("mult") = 1.0, py::arg("inject") = none, py::arg("inject_scale") = 1.0, py::arg("step") = none);
  m.def("softcap", [](Tensor& x, double cap) {
    TORCH_CHECK(x.is_cuda() && x.is_contiguous() && x.scalar_type() == at::kFloat, "softcap: contiguous fp32 CUDA tensor");
    check_rc(mb_softcap(x.data_ptr<float>(), x.numel(), static_cast<float>(cap), cur_stream()), "softcap");
  });
  m.def("gelu_tanh", [](Tensor& x) {
    TORCH_CHECK(x.is_cuda() && x.is_contiguous(), "gelu_tanh: contiguous CUDA tensor");
    check_rc(mb_gelu_tanh(x.data_ptr(), x.numel(), dtype_of(x, "x"), cur_stream()), "gelu_tanh");
  });
  m.def("sigmoid_gate", [](Tensor& o, const Tensor& g, int cols) {
    const int ldo = ld_of(o, o.scalar_type(), "o"), ldg = ld_of(g, o.scalar_type(), "g");
    TORCH_CHECK(o.size(1) >= cols && g.size(1) >= cols && g.size(0) >= o.size(0), "sigmoid_gate shapes");
    check_rc(mb_sigmoid_gate(o.data_ptr(), ldo, g.data_ptr(), ldg, o.size(0), cols, dtype_of(o, "o"), cur_stream()), "sigmoid_gate");
  });
  m.def("latent_post_down", &latent_post_down);
  m.def("rotate_heads", [](Tensor& x, int heads, int head_stride, int dims, bool interleaved, const Tensor& positions,
                           const Tensor& cos_sin) {
    const int ld = ld_of(x, x.scalar_type(), "x");
    TORCH_CHECK(static_cast<int64_t>(heads - 1) * head_stride + dims <= x.size(1) && cos_sin.dim() == 2 && cos_sin.size(1) == dims,
                "rotate_heads shapes");
    check_rc(mb_rotate_heads(x.data_ptr(), ld, x.size(0), heads, head_stride, dims, interleaved ? 1 : 0,
                             i32(positions, x.size(0), "positions"), f32(cos_sin, 0, "cos_sin"), dtype_of(x, "x"), cur_stream()),
             "rotate_heads");
  });
  m.def("latent_attention", &latent_attention, py::arg("q_lat"), py::arg("q_rope"), py::arg("cache"), py::arg("block_table"),
        py::arg("q_start"), py::arg("q_len"), py::arg("kv_len"), py::arg("out"), py::arg("scale"), py::arg("sink") = none,
        py::arg("one_token") = false, py::arg("ws") = none, py::arg("allow_tc") = true, py::arg("window") = 0,
        py::arg("gate") = none, py::arg("gate_mult") = 1.0);
  m.def("block_prep", &block_prep, py::arg("x"), py::arg("q_off"), py::arg("heads"), py::arg("k_off"), py::arg("v_off"),
        py::arg("kv_heads"), py::arg("dims"), py::arg("positions"), py::arg("cos_sin"), py::arg("slots"), py::arg("kv"), py::arg("plane"),
        py::arg("silu_off") = 0, py::arg("silu_n") = 0, py::arg("relu2_off") = 0, py::arg("relu2_n") = 0, py::arg("q_norm") = none,
        py::arg("k_norm") = none, py::arg("norm_dim") = 0, py::arg("eps") = 1e-6, py::arg("halves") = false,
        py::arg("bias") = none);
  m.def("window_attention", &window_attention, py::arg("q"), py::arg("out"), py::arg("kv"), py::arg("plane"), py::arg("block_table"),
        py::arg("q_start"), py::arg("q_len"), py::arg("kv_len"), py::arg("tile_seq"), py::arg("tile_q0"), py::arg("decode_seq"),
        py::arg("n_q"), py::arg("n_kv"), py::arg("scale"), py::arg("window") = 0, py::arg("sink") = none, py::arg("gate") = none,
        py::arg("gate_mult") = 1.0);
  m.def("attention_plan", [](const Tensor& q_len, int tok_per_tile, Tensor& tile_seq, Tensor& tile_q0) {
    const int n = tile_seq.numel();
    check_rc(mb_attention_plan(i32(q_len, 1, "q_len"), q_len.numel(), tok_per_tile, n,
                               const_cast<int32_t*>(i32(tile_seq, n, "tile_seq")), const_cast<int32_t*>(i32(tile_q0, n, "tile_q0")),
                               cur_stream()), "attention_plan");
  });
  m.def("lightning", &lightning);
  m.def("lightning_norm", [](Tensor& o, const Tensor& gate, const Tensor& w, int cols, int n, double eps) {
    const int ldo = ld_of(o, o.scalar_type(), "o"), ldg = ld_of(gate, o.scalar_type(), "gate");
    TORCH_CHECK(o.size(1) >= cols && gate.size(1) >= cols && gate.size(0) >= o.size(0) && w.is_contiguous() && w.numel() >= cols &&
                    w.scalar_type() == o.scalar_type(), "lightning_norm shapes");
    check_rc(mb_lightning_norm(o.data_ptr(), ldo, gate.data_ptr(), ldg, w.data_ptr(), o.size(0), cols, n, static_cast<float>(eps),
                               dtype_of(o, "o"), cur_stream()), "lightning_norm");
  });
  m.def("delta_dim_pad", [](int dim) { return mb_delta_dim_pad(dim); });
  m.def("delta_rule", &delta_rule, py::arg("x"), py::arg("q_off"), py::arg("k_off"), py::arg("v_off"), py::arg("b_off"), py::arg("conv_w"),
        py::arg("z"), py::arg("A_log"), py::arg("dt_bias"), py::arg("gate"), py::arg("norm_w"), py::arg("eps"), py::arg("scratch"),
        py::arg("out"), py::arg("state"), py::arg("conv_state"), py::arg("state_idx"), py::arg("q_start"), py::arg("q_len"),
        py::arg("kv_len"), py::arg("heads"), py::arg("kv_heads"), py::arg("dim"), py::arg("vdim"), py::arg("one_token"),
        py::arg("a_off") = -1, py::arg("gate_silu") = false, py::arg("out_mult") = 1.0);
  m.def("gla", &gla, py::arg("x"), py::arg("q_off"), py::arg("k_off"), py::arg("v_off"), py::arg("z"), py::arg("z_bias"), py::arg("q_scale"),
        py::arg("inv_tau"), py::arg("gate"), py::arg("gate_silu"), py::arg("out_mult"), py::arg("norm_w"), py::arg("eps"), py::arg("norm_dim"),
        py::arg("o"), py::arg("out"), py::arg("state"), py::arg("state_idx"), py::arg("q_start"), py::arg("q_len"), py::arg("kv_len"),
        py::arg("heads"), py::arg("dim"), py::arg("vdim"), py::arg("one_token"), py::arg("allow_chunks") = true);
  m.def("sandwich_norm", &sandwich_norm);
  m.def("tanh_seam", &tanh_seam);
  m.def("general_delta", &general_delta);
  m.def("tanh_cols", [](Tensor& x) {
    const int ld = ld_of(x, x.scalar_type(), "x");
    check_rc(mb_tanh_cols(x.data_ptr(), ld, x.size(0), x.size(1), dtype_of(x, "x"), cur_stream()), "tanh_cols");
  });
  m.def("xielu", [](Tensor& x, double up, double down) {
    const int ld = ld_of(x, x.scalar_type(), "x");
    check_rc(mb_xielu(x.data_ptr(), ld, x.size(0), x.size(1), static_cast<float>(up), static_cast<float>(down), dtype_of(x, "x"),
                      cur_stream()), "xielu");
  });
  m.def("bigram_rows", [](const Tensor& tokens, const Tensor& q_start, const Tensor& q_len, const Tensor& kv_len, const Tensor& state_idx,
                          Tensor& last, Tensor& out, int64_t mul_prev, int64_t mul_cur, int64_t buckets) {
    const int T = tokens.numel(), B = q_len.numel();
    TORCH_CHECK(tokens.is_cuda() && tokens.is_contiguous() && tokens.scalar_type() == at::kLong && last.is_cuda() && last.is_contiguous() &&
                    last.scalar_type() == at::kLong && out.is_cuda() && out.is_contiguous() && out.scalar_type() == at::kLong &&
                    out.numel() >= T, "bigram_rows: int64 CUDA tensors");
    check_rc(mb_bigram_rows(tokens.data_ptr<int64_t>(), i32(q_start, B, "q_start"), i32(q_len, B, "q_len"), i32(kv_len, B, "kv_len"),
                            i32(state_idx, B, "state_idx"), last.data_ptr<int64_t>(), out.data_ptr<int64_t>(), T, B, mul_prev, mul_cur,
                            buckets, cur_stream()), "bigram_rows");
  });
  m.def("moe_score_route", [](const Tensor& logits, const Opt& bias, Tensor& ids, Tensor& w, Tensor& rank, Tensor& counts, int n_group,
                              int keep, bool norm_topk, double scaling, bool softmax, bool group_max, int identity) {
    const int T = ids.size(0), k = ids.size(1), E = counts.numel() + identity, ld = ld_of(logits, at::kFloat, "logits");
    TORCH_CHECK(ids.dim() == 2 && logits.size(0) >= T && logits.size(1) >= E, "moe_score_route shapes");
    check_rc(mb_moe_score_route(logits.data_ptr<float>(), ld, given(bias) ? f32(*bias, E, "bias") : nullptr,
                                const_cast<int32_t*>(i32(ids, 0, "ids")), const_cast<float*>(f32(w, static_cast<int64_t>(T) * k, "w")),
                                const_cast<int32_t*>(i32(rank, static_cast<int64_t>(T) * k, "rank")),
                                const_cast<int32_t*>(i32(counts, E - identity, "counts")), T, E, n_group, keep, k, norm_topk ? 1 : 0,
                                static_cast<float>(scaling), softmax ? 1 : 0, group_max ? 1 : 0, identity, cur_stream()),
             "moe_score_route");
  }, py::arg("logits"), py::arg("bias"), py::arg("ids"), py::arg("w"), py::arg("rank"), py::arg("counts"), py::arg("n_group"),
     py::arg("keep"), py::arg("norm_topk"), py::arg("scaling"), py::arg("softmax") = false, py::arg("group_max") = false,
     py::arg("identity") = 0);
  m.def("moe_place_rows", [](const Tensor& x, const Tensor& ids, const Tensor& rank, const Tensor& counts, Tensor& offsets, Tensor& inverse,
                             Tensor& dst) {
    const int T = ids.size(0), k = ids.size(1), E = counts.numel(), es = x.element_size();
    const int ld = ld_of(x, x.scalar_type(), "x");
    TORCH_CHECK(dst.is_cuda() && dst.is_contiguous() && dst.dim() == 2 && dst.size(1) == x.size(1) && dst.scalar_type() == x.scalar_type() &&
                    dst.size(0) >= static_cast<int64_t>(T) * k && x.size(0) >= T, "moe_place_rows shapes");
    check_rc(mb_moe_place_rows(x.data_ptr(), static_cast<long long>(ld) * es, i32(ids, static_cast<int64_t>(T) * k, "ids"),
                               i32(rank, static_cast<int64_t>(T) * k, "rank"), i32(counts, E, "counts"),
                               const_cast<int32_t*>(i32(offsets, E + 1, "offsets")),
                               const_cast<int32_t*>(i32(inverse, static_cast<int64_t>(T) * k, "inverse")), dst.data_ptr(), T, E, k,
                               static_cast<int>(x.size(1)) * es, cur_stream()), "moe_place_rows");
  });
  m.def("moe_table_route", [](const Tensor& ids, const Tensor& tables, const Tensor& desc, int max_experts, Tensor& inverse,
                              Tensor& offsets) {
    TORCH_CHECK(ids.is_cuda() && ids.is_contiguous() && ids.scalar_type() == at::kLong && desc.is_cuda() && desc.is_contiguous() &&
                    desc.scalar_type() == at::kLong && desc.dim() == 2 && desc.size(1) == 6, "moe_table_route layout");
    check_rc(mb_moe_table_route(ids.data_ptr<int64_t>(), ids.numel(), i32(tables, 0, "tables"), desc.data_ptr<int64_t>(),
                                desc.size(0), max_experts, const_cast<int32_t*>(i32(inverse, 0, "inverse")),
                                const_cast<int32_t*>(i32(offsets, 0, "offsets")), cur_stream()),
             "moe_table_route");
  });
  m.def("gemm_f32", [](const Tensor& x, const Tensor& w, Tensor& y, const Opt& r) {
    const int ldx = ld_of(x, at::kFloat, "x"), ldw = ld_of(w, at::kFloat, "w"), ldy = ld_of(y, at::kFloat, "y");
    TORCH_CHECK(w.size(1) == x.size(1) && y.size(0) == x.size(0) && y.size(1) == w.size(0), "gemm_f32 shapes");
    int ldr = 0;
    if (given(r)) { ldr = ld_of(*r, at::kFloat, "residual"); TORCH_CHECK(r->sizes() == y.sizes(), "gemm_f32 residual"); }
    check_rc(mb_gemm_f32(x.data_ptr<float>(), w.data_ptr<float>(), y.data_ptr<float>(), static_cast<const float*>(optptr(r)),
                         x.size(0), w.size(0), x.size(1), ldx, ldw, ldy, ldr, cur_stream()), "gemm_f32");
  }, py::arg("x"), py::arg("w"), py::arg("y"), py::arg("residual") = none);
  m.def("batched_gemm_f32", [](const Tensor& x, const Tensor& w, Tensor& y, int x_off, int y_off) {
    const int ldx = ld_of(x, at::kFloat, "x"), ldy = ld_of(y, at::kFloat, "y");
    TORCH_CHECK(w.dim() == 3 && w.is_contiguous() && w.scalar_type() == at::kFloat, "batched_gemm_f32: w [B, N, K]");
    const int B = w.size(0), N = w.size(1), K = w.size(2);
    TORCH_CHECK(static_cast<int64_t>(B - 1) * x_off + K <= x.size(1) && static_cast<int64_t>(B - 1) * y_off + N <= y.size(1) &&
                    y.size(0) == x.size(0), "batched_gemm_f32: column blocks out of range");
    check_rc(mb_batched_gemm_f32(x.data_ptr<float>(), w.data_ptr<float>(), y.data_ptr<float>(), B, x.size(0), N, K, ldx, x_off,
                                 ldy, y_off, cur_stream()), "batched_gemm_f32");
  });
  m.def("grouped_gemm_f32", [](const Tensor& x, const Tensor& w, Tensor& y, const Tensor& offsets) {
    TORCH_CHECK(x.is_cuda() && x.is_contiguous() && w.is_contiguous() && y.is_contiguous() && w.dim() == 3 &&
                    x.scalar_type() == at::kFloat && w.scalar_type() == at::kFloat && y.scalar_type() == at::kFloat &&
                    x.size(1) == w.size(2) && y.size(1) == w.size(1) && y.size(0) == x.size(0), "grouped_gemm_f32 layout");
    check_rc(mb_grouped_gemm_f32(x.data_ptr<float>(), w.data_ptr<float>(), y.data_ptr<float>(), i32(offsets, w.size(0) + 1, "offsets"),
                                 w.size(0), x.size(0), w.size(1), w.size(2), cur_stream()), "grouped_gemm_f32");
  });
  m.def("silu_mul_f32", [](const Tensor& gu, Tensor& out) {
    TORCH_CHECK(gu.is_cuda() && gu.is_contiguous() && out.is_contiguous() && gu.scalar_type() == at::kFloat &&
                    out.scalar_type() == at::kFloat && gu.size(1) == 2 * out.size(1) && gu.size(0) == out.size(0), "silu_mul_f32");
    check_rc(mb_silu_mul_f32(gu.data_ptr<float>(), out.data_ptr<float>(), out.size(0), out.size(1), cur_stream()), "silu_mul_f32");
  });
}

// torch glue of the layer-stack kernels (stack.h): checks shapes, dtypes and strides, then hands over raw pointers.
#include <ATen/ATen.h>
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <torch/library.h>

#include <optional>

#include "kernels.h"
#include "runtime.h"
#include "stack.h"

namespace {

using at::Tensor;
using OptT = std::optional<Tensor>;

cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }
bool has(const OptT& t) { return t.has_value() && t->defined(); }

int* status_ptr(const Tensor& t) { return cosmos::status_tensor(t.get_device()).data_ptr<int>(); }

bool is_f32(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda(), name, " must be a CUDA tensor");
  TORCH_CHECK(t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat, name, " must be bfloat16 or float32");
  return t.scalar_type() == at::kFloat;
}
void check_i32(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kInt && t.is_contiguous(), name, " must be a contiguous int32 CUDA tensor");
}
const long long* i64_ptr(const Tensor& t, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kLong && t.is_contiguous(), name, " must be a contiguous int64 CUDA tensor");
  return reinterpret_cast<const long long*>(t.data_ptr<int64_t>());
}

// x [n, d] fp32 (updated in place); see ResidualNormArgs. y: [rows, >= d] of h's type, or fp32 partial sums
// [splits, rows, >= d]. h: [rows, >= d] or empty optional (sum only).
void residual_norm_(Tensor x, const OptT& embed, const OptT& tokens, double embed_scale, const OptT& y, const OptT& y_rows,
                    double weight, const OptT& gamma, int64_t groups, double eps, const OptT& h, const OptT& h_rows) {
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == at::kFloat && x.dim() == 2 && x.is_contiguous(), "x must be fp32 [n, d]");
  c10::cuda::CUDAGuard guard(x.device());
  cosmos::ResidualNormArgs a;
  const int64_t n = x.size(0), d = x.size(1);
  a.x = x.data_ptr<float>(); a.rows = n; a.d = (int)d;
  a.status = status_ptr(x);
  bool typed = false;
  auto set_type = [&](bool f32) {
    TORCH_CHECK(!typed || f32 == a.is_f32, "embed, gamma and h must have one dtype");
    a.is_f32 = f32;
    typed = true;
  };
  if (has(embed)) {
    TORCH_CHECK(has(tokens) && tokens->numel() == n && embed->dim() == 2 && embed->size(1) == d && embed->stride(1) == 1);
    set_type(is_f32(*embed, "embed"));
    a.embed = embed->data_ptr(); a.ld_embed = embed->stride(0); a.vocab = (int)embed->size(0);
    a.tokens = i64_ptr(*tokens, "tokens"); a.embed_scale = (float)embed_scale;
  }
  if (has(h)) {
    set_type(is_f32(*h, "h"));
    TORCH_CHECK(h->dim() == 2 && h->size(1) >= d && h->stride(1) == 1, "h must be [rows, >= d]");
    TORCH_CHECK(has(gamma) && gamma->is_contiguous() && gamma->numel() == d && gamma->scalar_type() == h->scalar_type(),
                "gamma must be [d] of h's type");
    a.gamma = gamma->data_ptr(); a.h = h->data_ptr(); a.ldh = h->stride(0); a.h_n = h->size(0);
    if (has(h_rows)) {
      check_i32(*h_rows, "h_rows");
      TORCH_CHECK(n > 0 && h_rows->numel() % n == 0);
      a.h_rows = h_rows->data_ptr<int>(); a.h_top = (int)(h_rows->numel() / n);
    } else {
      TORCH_CHECK(h->size(0) >= n);
    }
  }
  if (has(y)) {
    a.y_f32 = is_f32(*y, "y");
    if (!typed) set_type(a.y_f32);
    TORCH_CHECK(a.y_f32 || !a.is_f32, "a bf16 y needs bf16 outputs");
    TORCH_CHECK((y->dim() == 2 || (y->dim() == 3 && a.y_f32)) && y->size(-1) >= d && y->stride(-1) == 1, "bad y");
    a.y = y->data_ptr(); a.ldy = y->stride(-2); a.y_n = y->size(-2);
    if (y->dim() == 3) { a.k_splits = (int)y->size(0); a.split_stride = y->stride(0); }
    a.weight = (float)weight;
    if (has(y_rows)) {
      check_i32(*y_rows, "y_rows");
      TORCH_CHECK(n > 0 && y_rows->numel() % n == 0);
      a.y_rows = y_rows->data_ptr<int>(); a.top = (int)(y_rows->numel() / n);
    } else {
      TORCH_CHECK(y->size(-2) >= n);
    }
  }
  a.groups = (int)groups; a.eps = (float)eps;
  cosmos::residual_norm(a, cur_stream());
}

// Keys and normed / mixed values of n tokens into the cache; see QkvValueArgs. `qkv`: [n, >= cols] finished values, or
// fp32 partial sums [splits, n, >= cols] with `bias` (returns q [n, H, dim] then, else an empty tensor).
Tensor qkv_value_post(const Tensor& qkv, const OptT& bias, int64_t H, int64_t G, double eps, bool value_norm,
                      const Tensor& slots, Tensor k_cache, Tensor v_cache, const OptT& v_first_out, const OptT& v_first_in,
                      const OptT& lam) {
  c10::cuda::CUDAGuard guard(qkv.device());
  cosmos::QkvValueArgs a;
  a.is_f32 = is_f32(k_cache, "k_cache");
  TORCH_CHECK(k_cache.dim() == 4 && v_cache.dim() == 4 && k_cache.is_contiguous() && v_cache.is_contiguous() &&
                  v_cache.scalar_type() == k_cache.scalar_type() && k_cache.size(1) == G && v_cache.size(1) == G &&
                  k_cache.size(0) == v_cache.size(0) && k_cache.size(2) == v_cache.size(2),
              "caches must be contiguous [pages, G, page_size, head size] of one dtype");
  a.H = (int)H; a.G = (int)G; a.dim = (int)k_cache.size(3); a.vdim = (int)v_cache.size(3);
  a.page_size = (int)k_cache.size(2);
  a.k_cache = k_cache.data_ptr(); a.v_cache = v_cache.data_ptr();
  a.n_slots = k_cache.size(0) * k_cache.size(2);
  const int64_t cols = H * a.dim + G * (a.dim + a.vdim);
  const bool partial = qkv.dim() == 3;
  a.n = qkv.size(-2);
  TORCH_CHECK((qkv.dim() == 2 || partial) && qkv.size(-1) >= cols && qkv.stride(-1) == 1, "qkv must have q, k and v columns");
  Tensor q = at::empty({0}, k_cache.options());
  if (partial) {
    TORCH_CHECK(qkv.is_cuda() && qkv.scalar_type() == at::kFloat, "partial sums must be fp32");
    a.partial = qkv.data_ptr<float>(); a.k_splits = (int)qkv.size(0); a.split_stride = qkv.stride(0); a.ld_partial = qkv.stride(1);
    if (has(bias)) {
      TORCH_CHECK(bias->is_contiguous() && bias->numel() >= cols && bias->scalar_type() == k_cache.scalar_type(), "bad bias");
      a.bias = bias->data_ptr();
    }
    q = at::empty({a.n, H, a.dim}, k_cache.options());
    a.q_out = q.data_ptr();
  } else {
    TORCH_CHECK(qkv.is_cuda() && qkv.scalar_type() == k_cache.scalar_type(), "qkv must have the caches' dtype");
    a.qkv = qkv.data_ptr(); a.ld = qkv.stride(0);
  }
  a.eps = (float)eps; a.value_norm = value_norm;
  a.slots = i64_ptr(slots, "slots");
  TORCH_CHECK(slots.numel() == a.n, "one slot per token");
  for (const OptT* t : {&v_first_out, &v_first_in})
    if (has(*t))
      TORCH_CHECK((*t)->is_cuda() && (*t)->scalar_type() == at::kFloat && (*t)->is_contiguous() &&
                      (*t)->numel() == a.n * G * a.vdim, "first values must be fp32 [n, G, vdim]");
  if (has(v_first_out)) a.v_first_out = v_first_out->data_ptr<float>();
  if (has(v_first_in)) {
    TORCH_CHECK(has(lam) && lam->is_cuda() && lam->scalar_type() == at::kFloat && lam->numel() == 1, "lam must be one fp32 value");
    a.v_first_in = v_first_in->data_ptr<float>();
    a.lam = lam->data_ptr<float>();
  }
  a.status = status_ptr(k_cache);
  cosmos::qkv_value_post(a, cur_stream());
  return q;
}

// See WindowAttnArgs. q [n, H, dim] (unit inner stride, heads packed). tiles int32 [t, 4] of at most `tile_rows` rows, or
// none for a decode step (one query per sequence, at seq_lens - 1). impl: 0 = tcgen05 where it applies, 1 = CUDA cores.
Tensor window_attn(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& table, const OptT& seq_lens,
                   const OptT& tiles, int64_t tile_rows, double scale, int64_t window, const OptT& r1, const OptT& r2,
                   int64_t n_splits, int64_t impl) {
  c10::cuda::CUDAGuard guard(q.device());
  cosmos::WindowAttnArgs a;
  a.is_f32 = is_f32(q, "q");
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && q.stride(1) == q.size(2), "q must be [n, H, dim] with packed heads");
  TORCH_CHECK(k_cache.dim() == 4 && v_cache.dim() == 4 && k_cache.is_contiguous() && v_cache.is_contiguous() &&
                  k_cache.scalar_type() == q.scalar_type() && v_cache.scalar_type() == q.scalar_type() &&
                  k_cache.size(3) == q.size(2) && k_cache.size(0) == v_cache.size(0) && k_cache.size(1) == v_cache.size(1) &&
                  k_cache.size(2) == v_cache.size(2), "caches must be contiguous [pages, G, page_size, head size]");
  check_i32(table, "table");
  TORCH_CHECK(table.dim() == 2);
  a.q = q.data_ptr(); a.ldq = q.stride(0); a.n_rows = (int)q.size(0);
  a.H = (int)q.size(1); a.G = (int)k_cache.size(1); a.dim = (int)q.size(2); a.vdim = (int)v_cache.size(3);
  TORCH_CHECK(a.G > 0 && a.H % a.G == 0, "query heads must be a multiple of the key/value heads");
  a.k_cache = k_cache.data_ptr(); a.v_cache = v_cache.data_ptr();
  a.num_pages = (int)k_cache.size(0); a.page_size = (int)k_cache.size(2);
  a.table = table.data_ptr<int>(); a.max_pages = (int)table.size(1); a.n_seqs = (int)table.size(0);
  a.scale = (float)scale; a.window = (int)window;
  TORCH_CHECK(window >= 1, "window must be at least 1");
  auto per_head = [&](const OptT& t, const char* name) -> const float* {
    if (!has(t)) return nullptr;
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kFloat && t->is_contiguous() && t->numel() == a.H, name, " must be fp32 [H]");
    return t->data_ptr<float>();
  };
  a.r1 = per_head(r1, "r1");
  a.r2 = per_head(r2, "r2");   // none: a linear bias
  TORCH_CHECK(a.r1 || !a.r2, "r2 without r1");
  // a row is padded to a multiple of 8 elements: the output projection reads it with 16-byte rows
  const int64_t cols = (int64_t)a.H * a.vdim, ld = (cols + 7) / 8 * 8;
  Tensor out = at::empty({q.size(0), ld}, q.options());
  a.out = out.data_ptr(); a.ldo = ld;
  a.status = status_ptr(q);
  if (has(tiles)) {
    check_i32(*tiles, "tiles");
    TORCH_CHECK(tiles->dim() == 2 && tiles->size(1) == 4 && tile_rows > 0);
    a.tiles = tiles->data_ptr(); a.n_tiles = (int)tiles->size(0); a.tile_rows = (int)tile_rows;
    if (tile_rows <= cosmos::WINDOW_ATTN_SIMT_ROWS || impl == 1) {
      cosmos::window_attn_simt(a, cur_stream());
    } else {
      TORCH_CHECK(cosmos::window_attn_tc_supported(a), "window_attn: shape not supported by the tensor-core kernel");
      cosmos::window_attn_prefill_tc(a, cur_stream());
    }
    return out.narrow(1, 0, cols);
  }
  TORCH_CHECK(has(seq_lens), "a decode step needs seq_lens");
  check_i32(*seq_lens, "seq_lens");
  TORCH_CHECK(seq_lens->numel() == q.size(0) && table.size(0) == q.size(0), "one query row per sequence");
  a.seq_lens = seq_lens->data_ptr<int>();
  if (impl == 0 && cosmos::window_attn_decode_tc_supported(a)) {
    a.n_splits = (int)n_splits;
    Tensor ws;
    if (n_splits > 1) {
      a.scratch_bytes = cosmos::window_attn_scratch_bytes(a.n_seqs, a.H, a.vdim, a.n_splits);
      ws = at::empty({(int64_t)(a.scratch_bytes / 4)}, q.options().dtype(at::kFloat));
      a.scratch = ws.data_ptr<float>();
    }
    cosmos::window_attn_decode_tc(a, cur_stream());
  } else {
    cosmos::window_attn_simt(a, cur_stream());
  }
  return out.narrow(1, 0, cols);
}

// Whether the tcgen05 kernels take these shapes: (portions, decode).
std::tuple<bool, bool> window_attn_tc_supported(int64_t H, int64_t G, int64_t dim, int64_t vdim, int64_t page_size) {
  cosmos::WindowAttnArgs a;
  a.H = (int)H; a.G = (int)G; a.dim = (int)dim; a.vdim = (int)vdim; a.page_size = (int)page_size; a.num_pages = 1; a.ldq = 8;
  return {cosmos::window_attn_tc_supported(a), cosmos::window_attn_decode_tc_supported(a)};
}

int64_t window_attn_decode_splits(int64_t n_seqs, int64_t G, int64_t span) {
  return cosmos::window_attn_decode_splits((int)n_seqs, (int)G, (int)span);
}

// -> rows [layers, n * top_max] int32, tiles [layers, max_tiles, 4] int32, n_tiles [layers] int32
std::tuple<Tensor, Tensor, Tensor> moe_route(const Tensor& tokens, int64_t vocab, const Tensor& desc, int64_t max_experts,
                                             int64_t top_max, int64_t max_tiles) {
  c10::cuda::CUDAGuard guard(tokens.device());
  const long long* tok = i64_ptr(tokens, "tokens");
  const long long* de = i64_ptr(desc, "desc");
  TORCH_CHECK(desc.dim() == 2 && desc.size(1) == 4 && max_tiles >= 1 && top_max >= 1);
  const int64_t L = desc.size(0), n = tokens.numel();
  auto opt = tokens.options().dtype(at::kInt);
  Tensor rows = at::empty({L, n * top_max}, opt), tiles = at::empty({L, max_tiles, 4}, opt), cnt = at::empty({L}, opt);
  cosmos::moe_route(tok, n, (int)vocab, de, (int)L, (int)max_experts, (int)top_max, rows.data_ptr<int>(), tiles.data_ptr(),
                    (int)max_tiles, cnt.data_ptr<int>(), status_ptr(tokens), cur_stream());
  return {rows, tiles, cnt};
}

// Expert products over a tile map: a [R, K] rows sorted by expert, w [E, N, K] -> [R, N], or with `partial` the fp32 sums
// [k_splits, R, N] for a consumer that reduces them. gelu: exact gelu of the finished sum (not with `partial`).
Tensor grouped_gemm(const Tensor& a_, const Tensor& w, const Tensor& tiles, const Tensor& n_tiles, int64_t tile_m, bool gelu,
                    int64_t k_splits, bool partial) {
  c10::cuda::CUDAGuard guard(a_.device());
  const bool f32 = is_f32(a_, "a");
  TORCH_CHECK(w.is_cuda() && w.scalar_type() == a_.scalar_type() && w.dim() == 3 && w.stride(2) == 1 &&
                  w.stride(0) == w.size(1) * w.stride(1), "w must be [E, N, K] with evenly spaced rows");
  TORCH_CHECK(a_.dim() == 2 && a_.stride(1) == 1 && a_.size(1) == w.size(2), "a must be [R, K]");
  check_i32(tiles, "tiles"); check_i32(n_tiles, "n_tiles");
  TORCH_CHECK(tiles.dim() == 2 && tiles.size(1) == 4 && n_tiles.numel() == 1 && !(gelu && partial));
  const int64_t R = a_.size(0), N = w.size(1), K = w.size(2);
  if (f32) {
    TORCH_CHECK(tile_m == 128 && !partial, "the 32-bit product uses 128-row tiles and finishes its sums");
    Tensor c = at::empty({R, N}, a_.options());
    cosmos::grouped_gemm_f32(a_.data_ptr<float>(), a_.stride(0), w.data_ptr<float>(), w.stride(1), c.data_ptr<float>(), N,
                             (int)N, (int)K, tiles.data_ptr(), n_tiles.data_ptr<int>(), (int)tiles.size(0), gelu, cur_stream());
    return c;
  }
  TORCH_CHECK(N % 8 == 0 && a_.stride(0) % 8 == 0 && w.stride(1) % 8 == 0, "rows must be 16-byte aligned");
  cosmos::GemmArgs g;
  g.A = a_.data_ptr(); g.B = w.data_ptr();
  g.M = (int)R; g.N = (int)N; g.K = (int)K;
  g.lda = a_.stride(0); g.ldb = w.stride(1); g.ldc = N;
  g.epi = gelu ? EPI_GELU : EPI_PLAIN;
  g.status = status_ptr(a_);
  g.tile_map = tiles.data_ptr(); g.n_tiles_m = n_tiles.data_ptr<int>();
  g.n_groups = (int)w.size(0); g.max_tiles_m = (int)tiles.size(0); g.tile_m = (int)tile_m;
  Tensor c, part;
  if (!partial) {
    c = at::empty({R, N}, a_.options());
    g.C = c.data_ptr();
  }
  if (partial || k_splits > 1) {
    const int64_t k_blocks = (K + 63) / 64, ks = k_splits < 1 ? 1 : (k_splits < k_blocks ? k_splits : k_blocks);
    part = at::empty({ks, R, N}, a_.options().dtype(at::kFloat));
    g.k_splits = (int)ks; g.partial = part.data_ptr<float>(); g.partial_only = partial;
  }
  cosmos::gemm_bf16(g, cur_stream());
  return partial ? part : c;
}

// a [M, K] w [N, K]^T as fp32 partial sums [splits, M, N] (splits chosen for the machine; at least 1).
Tensor gemm_partial(const Tensor& a_, const Tensor& w) {
  c10::cuda::CUDAGuard guard(a_.device());
  TORCH_CHECK(!is_f32(a_, "a") && w.is_cuda() && w.scalar_type() == at::kBFloat16, "a and w must be bfloat16");
  TORCH_CHECK(a_.dim() == 2 && w.dim() == 2 && a_.stride(1) == 1 && w.stride(1) == 1 && a_.size(1) == w.size(1));
  TORCH_CHECK(w.size(0) % 8 == 0 && a_.stride(0) % 8 == 0 && w.stride(0) % 8 == 0, "rows must be 16-byte aligned");
  cosmos::GemmArgs g;
  g.A = a_.data_ptr(); g.B = w.data_ptr();
  g.M = (int)a_.size(0); g.N = (int)w.size(0); g.K = (int)w.size(1);
  g.lda = a_.stride(0); g.ldb = w.stride(0); g.ldc = g.N;
  g.epi = EPI_PLAIN;
  g.status = status_ptr(a_);
  g.k_splits = cosmos::gemm_pick_k_splits(g.M, g.N, g.K, g.epi);
  Tensor part = at::empty({g.k_splits, g.M, g.N}, a_.options().dtype(at::kFloat));
  g.partial = part.data_ptr<float>(); g.partial_only = true;
  cosmos::gemm_bf16(g, cur_stream());
  return part;
}

// ---------------------------------------------------------------- parallel layers and recurrent mixers
// Rows for a kernel of element type `f32 ? float : bf16`: finished values [n, >= cols] of that type, or fp32 values
// [n, >= cols] / split-K partial sums [splits, n, >= cols].
cosmos::RowSource row_source(const Tensor& t, bool f32, int64_t n, int64_t cols, const char* name) {
  TORCH_CHECK(t.is_cuda() && (t.dim() == 2 || t.dim() == 3) && t.stride(-1) == 1 && t.size(-2) >= n && t.size(-1) >= cols, name,
              " must be [n, cols] rows or [splits, n, cols] partial sums");
  cosmos::RowSource s;
  s.p = t.data_ptr(); s.ld = t.stride(-2);
  if (t.dim() == 2 && is_f32(t, name) == f32) return s;
  TORCH_CHECK(t.scalar_type() == at::kFloat, name, ": partial sums must be fp32");
  s.k_splits = t.dim() == 3 ? (int)t.size(0) : 1;
  s.split_stride = t.dim() == 3 ? t.stride(0) : 0;
  return s;
}
const float* f32_vec(const Tensor& t, int64_t n, const char* name) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() == n, name, " must be contiguous fp32 with ",
              n, " entries");
  return t.data_ptr<float>();
}
// portions int32 [p, 4], or lens int32 [n] of a decode step; state_slots int32 [sequences].
cosmos::StepRows step_rows(const OptT& portions, const OptT& lens, const Tensor& state_slots, int64_t n_rows, int64_t n_state_slots) {
  cosmos::StepRows r;
  check_i32(state_slots, "state_slots");
  r.state_slots = state_slots.data_ptr<int>();
  r.n_state_slots = (int)n_state_slots;
  if (has(portions)) {
    check_i32(*portions, "portions");
    TORCH_CHECK(portions->dim() == 2 && portions->size(1) == 4, "portions must be [p, 4]");
    r.portions = portions->data_ptr(); r.n = (int)portions->size(0);
  } else {
    TORCH_CHECK(has(lens), "a decode step needs lens");
    check_i32(*lens, "lens");
    TORCH_CHECK(lens->numel() == n_rows && state_slots.numel() == n_rows, "one row per sequence");
    r.lens = lens->data_ptr<int>(); r.n = (int)n_rows;
  }
  return r;
}
Tensor padded_rows(int64_t n, int64_t cols, const at::TensorOptions& o) {
  return at::empty({n, (cols + 7) / 8 * 8}, o).narrow(1, 0, cols);
}

// See BranchNormArgs. x [n, d] fp32 in place; `normed` up to two branches with their weights; h1 / h2 [n, >= d].
void branch_norm_(Tensor x, const OptT& embed, const OptT& tokens, double embed_scale, const OptT& pos_turns, const OptT& positions,
                  at::TensorList normed, at::TensorList normed_w, double coef, const OptT& plain, const OptT& gamma1, const OptT& gamma2,
                  double gamma_add, double eps, const OptT& h1, const OptT& h2, bool f32) {
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == at::kFloat && x.dim() == 2 && x.is_contiguous(), "x must be fp32 [n, d]");
  c10::cuda::CUDAGuard guard(x.device());
  cosmos::BranchNormArgs a;
  const int64_t n = x.size(0), d = x.size(1);
  a.x = x.data_ptr<float>(); a.rows = n; a.d = (int)d; a.is_f32 = f32;
  a.status = status_ptr(x);
  if (has(embed)) {
    TORCH_CHECK(has(tokens) && tokens->numel() == n && embed->dim() == 2 && embed->size(1) == d && embed->stride(1) == 1 &&
                is_f32(*embed, "embed") == f32);
    a.embed = embed->data_ptr(); a.ld_embed = embed->stride(0); a.vocab = (int)embed->size(0);
    a.tokens = i64_ptr(*tokens, "tokens"); a.embed_scale = (float)embed_scale;
    if (has(pos_turns)) {
      TORCH_CHECK(pos_turns->is_cuda() && pos_turns->scalar_type() == at::kDouble && pos_turns->is_contiguous() &&
                      pos_turns->numel() == (d + 1) / 2 && has(positions) && positions->numel() == n, "bad position table");
      a.pos_turns = pos_turns->data_ptr<double>();
      a.positions = i64_ptr(*positions, "positions");
    }
  }
  TORCH_CHECK(normed.size() <= 2 && normed.size() == normed_w.size(), "up to two normed branches with a weight each");
  a.n_normed = (int)normed.size(); a.coef = (float)coef;
  for (size_t i = 0; i < normed.size(); ++i) {
    a.normed[i] = row_source(normed[i], f32, n, d, "branch");
    a.normed_w[i] = f32_vec(normed_w[i], d, "branch weight");
  }
  if (has(plain)) {
    a.has_plain = true;
    a.plain = row_source(*plain, f32, n, d, "plain");
  }
  const OptT* hs[2] = {&h1, &h2};
  const OptT* gs[2] = {&gamma1, &gamma2};
  for (int i = 0; i < 2; ++i) {
    if (!has(*hs[i])) continue;
    const Tensor& h = **hs[i];
    TORCH_CHECK(has(*gs[i]) && is_f32(h, "h") == f32 && h.dim() == 2 && h.size(0) >= n && h.size(1) >= d && h.stride(1) == 1, "bad h");
    TORCH_CHECK(a.ldh == 0 || a.ldh == h.stride(0), "h1 and h2 must have one row stride");
    a.h[i] = h.data_ptr(); a.ldh = h.stride(0);
    a.gamma[i] = f32_vec(**gs[i], d, "gamma");
  }
  a.gamma_add = (float)gamma_add; a.eps = (float)eps;
  cosmos::branch_norm(a, cur_stream());
}

// See QkNormArgs -> q [n, H, dim]
Tensor qk_norm_post(const Tensor& q, const Tensor& k, int64_t H, int64_t G, const Tensor& wq, const Tensor& wk, double eps,
                    double temp_coef, int64_t temp_every, const Tensor& positions, const Tensor& slots, Tensor k_cache, Tensor v_cache) {
  c10::cuda::CUDAGuard guard(q.device());
  cosmos::QkNormArgs a;
  a.is_f32 = is_f32(k_cache, "k_cache");
  TORCH_CHECK(k_cache.dim() == 4 && k_cache.is_contiguous() && v_cache.is_contiguous() && v_cache.sizes() == k_cache.sizes() &&
                  v_cache.scalar_type() == k_cache.scalar_type() && k_cache.size(1) == G, "caches must be contiguous [pages, G, page_size, dim]");
  a.n = slots.numel(); a.H = (int)H; a.G = (int)G; a.dim = (int)k_cache.size(3);
  a.q = row_source(q, a.is_f32, a.n, H * a.dim, "q");
  a.k = row_source(k, a.is_f32, a.n, G * a.dim, "k");
  a.wq = f32_vec(wq, H * a.dim, "wq"); a.wk = f32_vec(wk, G * a.dim, "wk");
  a.eps = (float)eps; a.temp_coef = (float)temp_coef; a.temp_every = temp_every;
  TORCH_CHECK(positions.numel() == a.n, "one position per token");
  a.positions = i64_ptr(positions, "positions"); a.slots = i64_ptr(slots, "slots");
  a.n_slots = k_cache.size(0) * k_cache.size(2); a.page_size = (int)k_cache.size(2);
  a.k_cache = k_cache.data_ptr(); a.v_cache = v_cache.data_ptr();
  Tensor out = at::empty({a.n, H, a.dim}, k_cache.options());
  a.q_out = out.data_ptr();
  a.status = status_ptr(k_cache);
  cosmos::qk_norm_post(a, cur_stream());
  return out;
}

// See CausalConvArgs -> u [n, inner] (row stride padded to 8)
Tensor causal_conv(const Tensor& x, const Tensor& w, const Tensor& b, Tensor conv_state, const Tensor& state_slots,
                   const OptT& portions, const OptT& tiles, const OptT& lens, int64_t n) {
  c10::cuda::CUDAGuard guard(x.device());
  cosmos::CausalConvArgs a;
  TORCH_CHECK(w.dim() == 2 && conv_state.dim() == 3 && conv_state.is_contiguous() && conv_state.size(1) == w.size(1) - 1 &&
                  conv_state.size(2) == w.size(0), "conv_state must be [slots, taps - 1, inner]");
  a.is_f32 = is_f32(conv_state, "conv_state");
  a.inner = (int)w.size(0); a.taps = (int)w.size(1);
  a.x = row_source(x, a.is_f32, n, a.inner, "x");
  a.w = f32_vec(w, w.numel(), "w"); a.b = f32_vec(b, a.inner, "b");
  a.conv_state = conv_state.data_ptr();
  a.rows = step_rows(portions, lens, state_slots, n, conv_state.size(0));
  if (has(portions)) {
    TORCH_CHECK(has(tiles), "portions need their tiles");
    check_i32(*tiles, "tiles");
    TORCH_CHECK(tiles->dim() == 2 && tiles->size(1) == 8, "tiles must be [t, 8]");
    a.tiles = tiles->data_ptr<int>(); a.n_tiles = (int)tiles->size(0);
  }
  Tensor u = padded_rows(n, a.inner, conv_state.options());
  a.u = u.data_ptr(); a.ldu = u.stride(0);
  a.status = status_ptr(x);
  cosmos::causal_conv(a, cur_stream());
  return u;
}

// See SelectiveScanArgs. y [n, >= inner]: columns [0, inner) are written, and zeros into [inner, y_cols).
void selective_scan(const Tensor& u, const Tensor& dt, const Tensor& z, const Tensor& bc, const Tensor& dt_bias, const Tensor& a2,
                    const Tensor& D, Tensor S, Tensor y, int64_t y_cols, const Tensor& state_slots, const OptT& portions,
                    const OptT& lens) {
  c10::cuda::CUDAGuard guard(u.device());
  cosmos::SelectiveScanArgs a;
  a.is_f32 = is_f32(u, "u");
  const int64_t n = u.size(0);
  TORCH_CHECK(S.dim() == 3 && S.scalar_type() == at::kFloat && S.is_contiguous(), "S must be fp32 [slots, inner, state]");
  a.inner = (int)S.size(1); a.state = (int)S.size(2);
  TORCH_CHECK(u.dim() == 2 && u.size(1) == a.inner && u.stride(1) == 1 && is_f32(y, "y") == a.is_f32 && y.dim() == 2 &&
                  y.size(0) == n && y.stride(1) == 1 && y.size(1) >= y_cols && y_cols >= a.inner, "bad u or y");
  a.u = u.data_ptr(); a.ldu = u.stride(0);
  a.dt = row_source(dt, a.is_f32, n, a.inner, "dt");
  a.z = row_source(z, a.is_f32, n, a.inner, "z");
  a.bc = row_source(bc, a.is_f32, n, 2 * a.state, "bc");
  a.dt_bias = f32_vec(dt_bias, a.inner, "dt_bias");
  a.a2 = f32_vec(a2, (int64_t)a.inner * a.state, "a2");
  a.D = f32_vec(D, a.inner, "D");
  a.S = S.data_ptr<float>();
  a.y = y.data_ptr(); a.ldy = y.stride(0);
  a.rows = step_rows(portions, lens, state_slots, n, S.size(0));
  a.status = status_ptr(u);
  cosmos::selective_scan(a, cur_stream());
  cosmos::zero_cols(a.y, a.ldy, a.inner, (int)y_cols, n, a.is_f32, cur_stream());
}

// See MatrixMemoryArgs -> o [n, H * vdim] (row stride padded to 8). S [slots, H, dim, vdim], nrm [slots, H, slices, dim],
// m [slots, H, slices] fp32. impl 0 = tcgen05 where it applies, 1 = CUDA cores.
Tensor matrix_memory(const Tensor& q, const Tensor& k, const Tensor& v, const Tensor& gates, const Tensor& gate_bias, double q_scale,
                     double cap, Tensor S, Tensor nrm, Tensor m, const Tensor& state_slots, const OptT& portions, const OptT& lens,
                     int64_t n, bool f32, int64_t impl) {
  c10::cuda::CUDAGuard guard(q.device());
  cosmos::MatrixMemoryArgs a;
  TORCH_CHECK(S.dim() == 4 && S.scalar_type() == at::kFloat && S.is_contiguous(), "S must be fp32 [slots, H, dim, vdim]");
  a.is_f32 = f32;
  a.H = (int)S.size(1); a.dim = (int)S.size(2); a.vdim = (int)S.size(3);
  const int64_t slices = (a.vdim + cosmos::MEMORY_SLICE - 1) / cosmos::MEMORY_SLICE;
  a.S = S.data_ptr<float>();
  a.n = const_cast<float*>(f32_vec(nrm, S.size(0) * a.H * slices * a.dim, "nrm"));
  a.m = const_cast<float*>(f32_vec(m, S.size(0) * a.H * slices, "m"));
  a.q = row_source(q, f32, n, (int64_t)a.H * a.dim, "q");
  a.k = row_source(k, f32, n, (int64_t)a.H * a.dim, "k");
  a.v = row_source(v, f32, n, (int64_t)a.H * a.vdim, "v");
  TORCH_CHECK(gates.scalar_type() == at::kFloat, "gates must be fp32");
  a.gates = row_source(gates, true, n, 2 * a.H, "gates");
  a.gate_bias = f32_vec(gate_bias, 2 * a.H, "gate_bias");
  a.q_scale = (float)q_scale; a.cap = (float)cap;
  a.rows = step_rows(portions, lens, state_slots, n, S.size(0));
  Tensor o = padded_rows(n, (int64_t)a.H * a.vdim, S.options().dtype(f32 ? at::kFloat : at::kBFloat16));
  a.o = o.data_ptr(); a.ldo = o.stride(0);
  a.status = status_ptr(q);
  a.n_rows = n;
  // the chunked kernel once portions fill a good part of a chunk
  if (impl == 0 && n >= 48 * (int64_t)a.rows.n && cosmos::matrix_memory_tc_supported(a))
    cosmos::matrix_memory_tc(a, cur_stream());
  else
    cosmos::matrix_memory(a, cur_stream());
  return o;
}

// y = o / rms(head of o) * w * sigmoid(g), heads of w.numel() / H columns
Tensor head_norm_gate(const Tensor& o, const Tensor& g, const Tensor& w, int64_t H, double eps) {
  c10::cuda::CUDAGuard guard(o.device());
  cosmos::HeadNormGateArgs a;
  a.is_f32 = is_f32(o, "o");
  const int64_t cols = w.numel();
  TORCH_CHECK(o.dim() == 2 && o.size(1) == cols && o.stride(1) == 1 && H > 0 && cols % H == 0, "o must be [n, H * vdim]");
  a.o = o.data_ptr(); a.ldo = o.stride(0); a.n = o.size(0); a.H = (int)H; a.vdim = (int)(cols / H);
  a.g = row_source(g, a.is_f32, a.n, cols, "g");
  a.w = f32_vec(w, cols, "w"); a.eps = (float)eps;
  Tensor y = padded_rows(a.n, cols, o.options());
  a.y = y.data_ptr(); a.ldy = y.stride(0);
  cosmos::head_norm_gate(a, cur_stream());
  return y;
}

}  // namespace

TORCH_LIBRARY_FRAGMENT(cosmos_b200, m) {
  m.def("residual_norm_", &residual_norm_);
  m.def("qkv_value_post", &qkv_value_post);
  m.def("window_attn", &window_attn);
  m.def("window_attn_tc_supported", &window_attn_tc_supported);
  m.def("window_attn_decode_splits", &window_attn_decode_splits);
  m.def("moe_route", &moe_route);
  m.def("grouped_gemm", &grouped_gemm);
  m.def("gemm_partial", &gemm_partial);
  m.def("branch_norm_", &branch_norm_);
  m.def("qk_norm_post", &qk_norm_post);
  m.def("causal_conv", &causal_conv);
  m.def("selective_scan", &selective_scan);
  m.def("matrix_memory", &matrix_memory);
  m.def("head_norm_gate", &head_norm_gate);
}

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
  if (has(r1)) {
    TORCH_CHECK(has(r2) && r1->is_cuda() && r2->is_cuda() && r1->scalar_type() == at::kFloat && r2->scalar_type() == at::kFloat &&
                    r1->is_contiguous() && r2->is_contiguous() && r1->numel() == a.H && r2->numel() == a.H, "r1, r2 must be fp32 [H]");
    a.r1 = r1->data_ptr<float>(); a.r2 = r2->data_ptr<float>();
  }
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
}

// Launchers of the kernels behind config-declared layer stacks (models/stack.py): a 32-bit residual stream, grouped
// RMS norms, value norm / value mixing, windowed attention with a distance bias over the paged cache, and experts
// chosen by a token table. Element type: bf16 (is_f32 = false) or fp32.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace cosmos {

// One pass per token row over the residual stream x (fp32):
//   x  = embed[token] * embed_scale            (embed != null), else x as it is
//   x += weight * sum_{k < top} sum_{s < k_splits} y[s][row_k]      (y != null; row_k = y_rows[row * top + k] or row)
//   h  = gamma * (x in `groups` parts, each divided by its own root mean square)
// h goes to row `row`, or to the rows h_rows[row * h_top + k] (the expert-sorted buffer of the next feed-forward).
struct ResidualNormArgs {
  float* x = nullptr;
  long long rows = 0;
  int d = 0;
  const void* embed = nullptr;
  long long ld_embed = 0;
  const long long* tokens = nullptr;
  int vocab = 0;
  float embed_scale = 1.f;
  const void* y = nullptr;
  bool y_f32 = false;
  int k_splits = 1;
  long long split_stride = 0, ldy = 0, y_n = 0;  // y_n: rows of y
  const int* y_rows = nullptr;
  int top = 1;
  float weight = 1.f;
  const void* gamma = nullptr;
  int groups = 1;
  float eps = 1e-6f;
  void* h = nullptr;
  long long ldh = 0, h_n = 0;
  const int* h_rows = nullptr;
  int h_top = 1;
  bool is_f32 = false;
  int* status = nullptr;
};
void residual_norm(const ResidualNormArgs& a, cudaStream_t s);

// After the q/k/v projection. qkv rows: [H * dim | G * dim | G * vdim]; either finished values (type T, row stride ld) or
// split-K partial sums [k_splits][n][ncols] (fp32) to which the bias is added here. Keys go into their cache rows; every
// value head is divided by its root mean square, mixed with the values of an earlier layer (v <- (1 - lam) v + lam v0)
// and cached. q is written to q_out [n, H, dim] only from partial sums.
struct QkvValueArgs {
  const void* qkv = nullptr;
  long long ld = 0;
  const float* partial = nullptr;
  int k_splits = 1;
  long long split_stride = 0, ld_partial = 0;
  const void* bias = nullptr;
  long long n = 0;
  int H = 0, G = 0, dim = 0, vdim = 0;
  float eps = 1e-6f;
  bool value_norm = true;
  const long long* slots = nullptr;
  long long n_slots = 0;
  void* q_out = nullptr;
  void* k_cache = nullptr;   // [pages, G, page_size, dim]
  void* v_cache = nullptr;   // [pages, G, page_size, vdim]
  int page_size = 0;
  float* v_first_out = nullptr;       // [n, G, vdim]: this layer's values, for later layers
  const float* v_first_in = nullptr;
  const float* lam = nullptr;         // device scalar
  bool is_f32 = false;
  int* status = nullptr;
};
void qkv_value_post(const QkvValueArgs& a, cudaStream_t s);

// Attention of new tokens over the paged cache: query at position i sees keys 0 <= i - j < window, score =
// scale * q.k - r1[h] * ln(1 + r2[h] * (i - j)), softmax, weighted sum of the values.
//   tiles: int4 {sequence, first query row, rows, position of the first row} (device), at most `tile_rows` rows each;
//          null: sequence b has the one query row b at position seq_lens[b] - 1 (a decode step; length 0 = idle)
//   table [n_seqs, max_pages]; q row stride ldq, head h at h * dim; out row stride ldo, head h at h * vdim.
// r2 null: the bias is linear, r1[h] * (i - j).
struct WindowAttnArgs {
  const void* q = nullptr;
  long long ldq = 0;
  const void* k_cache = nullptr;
  const void* v_cache = nullptr;
  const int* table = nullptr;
  int max_pages = 0, num_pages = 0, page_size = 0;
  const int* seq_lens = nullptr;
  const void* tiles = nullptr;
  int n_tiles = 0, tile_rows = 0;
  int n_rows = 0;           // rows of q
  int n_seqs = 0;
  int H = 0, G = 0, dim = 0, vdim = 0;
  float scale = 1.f;
  int window = 0;
  const float* r1 = nullptr;   // [H]; null = no bias
  const float* r2 = nullptr;
  void* out = nullptr;
  long long ldo = 0;
  bool is_f32 = false;
  // decode on the tensor cores: splits of the window and their partial sums (see paged_decode.cu)
  int n_splits = 1;
  float* scratch = nullptr;
  size_t scratch_bytes = 0;
  int* status = nullptr;
};
// CUDA-core kernel: any head sizes up to 512, bf16 or fp32; portions (16-row tiles) and decode steps.
constexpr int WINDOW_ATTN_SIMT_ROWS = 16;
void window_attn_simt(const WindowAttnArgs& a, cudaStream_t s);
// tcgen05 kernels (bf16, head sizes up to 128 that are multiples of 8, pages of 8 .. 128 tokens).
constexpr int WINDOW_ATTN_TC_ROWS = 256;
bool window_attn_tc_supported(const WindowAttnArgs& a);
void window_attn_prefill_tc(const WindowAttnArgs& a, cudaStream_t s);
bool window_attn_decode_tc_supported(const WindowAttnArgs& a);   // also needs a GQA group of 1, 2, 4 or 8
int window_attn_decode_splits(int n_seqs, int G, int span);
size_t window_attn_scratch_bytes(int n_seqs, int H, int vdim, int n_splits);
void window_attn_decode_tc(const WindowAttnArgs& a, cudaStream_t s);

// Routing of a step for `n_layers` layers at once: desc [n_layers, 4] int64 (device) = {address of the layer's int32
// table [vocab, top], experts, top, rows per tile}. Per layer: rows[n * top] = place of (token, k) in expert order
// (layer stride n * top_max), tiles = {expert, first row, rows, 0} per m-tile (layer stride max_tiles), n_tiles.
void moe_route(const long long* tokens, long long n, int vocab, const long long* desc, int n_layers, int max_experts,
               int top_max, int* rows, void* tiles, int max_tiles, int* n_tiles, int* status, cudaStream_t s);

// fp32 grouped GEMM over a tile map of 128-row tiles: C[r] = act(A[r] W_group^T), W [groups * N, K].
void grouped_gemm_f32(const float* A, long long lda, const float* W, long long ldw, float* C, long long ldc, int N, int K,
                      const void* tiles, const int* n_tiles, int max_tiles, int gelu, cudaStream_t s);

// ---------------------------------------------------------------- rows, portions and state of a step
// [n, cols] rows with unit column stride: finished values of the launch's element type (k_splits = 0), or fp32 split-K
// partial sums [k_splits][n][cols] that the reader adds up.
struct RowSource {
  const void* p = nullptr;
  int k_splits = 0;
  long long split_stride = 0, ld = 0;
};
// The tokens of a step as recurrent layers see them. portions: int4 {sequence, first row, rows, position of the first row}
// (device); null: sequence b has the one row b at position lens[b] - 1 (a decode step; length 0 = idle, its state is left
// alone). state_slots [sequences]: where a sequence's state lives. A sequence at position 0 starts from a zero state, so a
// slot needs no clearing before it is used again.
struct StepRows {
  const void* portions = nullptr;
  const int* lens = nullptr;
  const int* state_slots = nullptr;
  int n = 0, n_state_slots = 0;
};

// Parallel layers: x += coef * sum_b (y_b / rms(y_b) * w_b) (up to two normed branches) + y_plain, then two norms of the same
// x: h_i = x / rms(x) * (gamma_add + gamma_i). With `embed`, x starts as embed[token] * embed_scale, plus (pos_turns != null)
// the sinusoid of the position: entry 2i sin(2 pi p turns_i), entry 2i + 1 the cosine.
struct BranchNormArgs {
  float* x = nullptr;
  long long rows = 0;
  int d = 0;
  const void* embed = nullptr;
  long long ld_embed = 0;
  const long long* tokens = nullptr;
  int vocab = 0;
  float embed_scale = 1.f;
  const double* pos_turns = nullptr;   // [(d + 1) / 2] turns per position
  const long long* positions = nullptr;
  int n_normed = 0;
  RowSource normed[2];
  const float* normed_w[2] = {nullptr, nullptr};
  float coef = 1.f;
  bool has_plain = false;
  RowSource plain;
  const float* gamma[2] = {nullptr, nullptr};
  void* h[2] = {nullptr, nullptr};     // null = not wanted
  float gamma_add = 0.f;
  long long ldh = 0;
  float eps = 1e-6f;
  bool is_f32 = false;
  int* status = nullptr;
};
void branch_norm(const BranchNormArgs& a, cudaStream_t s);

// Queries and keys normed over the whole projection (all heads at once) with weights wq / wk, queries times
// 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1); keys go into the cache, and the projected keys before the norm go
// into the value cache (the values are the keys).
struct QkNormArgs {
  RowSource q, k;
  long long n = 0;
  int H = 0, G = 0, dim = 0;
  const float* wq = nullptr;
  const float* wk = nullptr;
  float eps = 1e-6f, temp_coef = 0.f;
  long long temp_every = 0;            // 0 = no temperature
  const long long* positions = nullptr;
  const long long* slots = nullptr;
  long long n_slots = 0;
  void* q_out = nullptr;               // [n, H * dim]
  void* k_cache = nullptr;             // [pages, G, page_size, dim]
  void* v_cache = nullptr;
  int page_size = 0;
  bool is_f32 = false;
  int* status = nullptr;
};
void qk_norm_post(const QkNormArgs& a, cudaStream_t s);

// ---------------------------------------------------------------- selective scan (selective_scan.cu)
// Causal convolution per channel + silu: u[t] = silu(b + sum_j w[c, j] x[t - (taps - 1 - j)]); inputs before the portion come
// from conv_state [slots, taps - 1, inner] (oldest first), which ends up holding the portion's last taps - 1 inputs.
// tiles (portions only): int32 [n_tiles][8] = sequence, first row, rows, position of the portion's first row, portion's first row.
struct CausalConvArgs {
  RowSource x;
  int inner = 0, taps = 0;
  const float* w = nullptr;            // [inner, taps]
  const float* b = nullptr;            // [inner]
  void* conv_state = nullptr;
  void* u = nullptr;
  long long ldu = 0;
  StepRows rows;
  const int* tiles = nullptr;
  int n_tiles = 0;
  bool is_f32 = false;
  int* status = nullptr;
};
constexpr int CONV_TILE_ROWS = 32;
constexpr int CONV_MAX_TAPS = 16;
void causal_conv(const CausalConvArgs& a, cudaStream_t s);

// S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n; y_c = (sum_n S[c, n] C_n + D_c u_c) silu(z_c), with
// dt = softplus(dt_raw + dt_bias). a2 = A log2(e).
struct SelectiveScanArgs {
  RowSource dt, z, bc;                 // bc: B in columns [0, state), C in [state, 2 state)
  const void* u = nullptr;
  long long ldu = 0;
  int inner = 0, state = 0;
  const float* dt_bias = nullptr;
  const float* a2 = nullptr;           // [inner, state]
  const float* D = nullptr;
  float* S = nullptr;                  // [slots, inner, state]
  void* y = nullptr;
  long long ldy = 0;
  StepRows rows;
  bool is_f32 = false;
  int* status = nullptr;
};
constexpr int SCAN_MAX_STATE = 128;
void selective_scan(const SelectiveScanArgs& a, cudaStream_t s);
// Zeros into columns [c0, c1) of y [n, >= c1].
void zero_cols(void* y, long long ldy, int c0, int c1, long long n, bool is_f32, cudaStream_t s);

// ---------------------------------------------------------------- matrix memory (matrix_memory.cu)
// mLSTM: log gates i = cap tanh((i_raw + i_b) / cap), f = logsigmoid(cap tanh((f_raw + f_b) / cap)); running maximum
// m_t = max(f + m, i) from 0; S = exp(f + m_(t-1) - m) S + exp(i - m) k v^T, n likewise with k;
// o = S^T q / (max(|n . q|, exp(-m)) + 1e-6), q scaled by q_scale.
// State: S [slots, H, dim, vdim]; n [slots, H, slices, dim] and m [slots, H, slices], one copy for every MEMORY_SLICE
// value columns, so that the CTAs of a head share nothing.
struct MatrixMemoryArgs {
  RowSource q, k, v, gates;            // gates: H columns of i_raw, then H of f_raw
  int H = 0, dim = 0, vdim = 0;
  float q_scale = 1.f, cap = 1.f;
  const float* gate_bias = nullptr;    // [2 H]
  float* S = nullptr;
  float* n = nullptr;
  float* m = nullptr;
  void* o = nullptr;                   // [n_rows, H * vdim]
  long long ldo = 0, n_rows = 0;
  StepRows rows;
  bool is_f32 = false;
  int* status = nullptr;
};
constexpr int MEMORY_SLICE = 32;
constexpr int MEMORY_MAX_DIM = 512;
void matrix_memory(const MatrixMemoryArgs& a, cudaStream_t s);      // CUDA cores: any sizes, bf16 or fp32, portions and decode steps
// tcgen05, chunks of 128 tokens (matrix_memory_tc.cu): bf16 portions, dim 64 / 128 / 256, vdim a multiple of MEMORY_SLICE.
bool matrix_memory_tc_supported(const MatrixMemoryArgs& a);
void matrix_memory_tc(const MatrixMemoryArgs& a, cudaStream_t s);

// y = o / rms(o of the head) * w * sigmoid(g)
struct HeadNormGateArgs {
  const void* o = nullptr;
  long long ldo = 0;
  RowSource g;
  const float* w = nullptr;            // [H * vdim]
  long long n = 0;
  int H = 0, vdim = 0;
  float eps = 1e-6f;
  void* y = nullptr;
  long long ldy = 0;
  bool is_f32 = false;
};
void head_norm_gate(const HeadNormGateArgs& a, cudaStream_t s);

}  // namespace cosmos

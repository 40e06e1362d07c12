// torch.ops.omni_b200.* : the ops of the core library (_C_core.so), which every model needs (matrix
// products, routing, sampling) or which a model can run on without the rest (attention with a window,
// sink and gate, the 32-bit residual stream).  The other ops are in bindings.cpp (_C.so, linked
// against this library).  Tensors are validated here; the kernels are plain C launchers.

#include <tuple>

#include "bindings_common.h"

extern "C" {
void b200_gemm_plan(int M, int N, int K, int elem_bytes, int swiglu, int force_bn, int force_splits,
                    int* out_bn, int* out_splits, size_t* out_ws_bytes, int* out_counters,
                    int* out_cluster);
int b200_gemm(const void* A, const void* W, void* C, const void* bias, const void* residual, int M,
              int N, int K, int lda, int ldw, int ldc, int dtype_fp8, int out_fp32, int swiglu,
              int BN, int splits, int cluster_split, void* workspace, int* counters, int* status,
              int max_ctas, float act_alpha, float act_limit, cudaStream_t stream);
int b200_gemm_pair(const void* A, const void* W, void* C, const void* bias, const void* residual,
                   int M, int N, int K, int lda, int ldw, int ldc, int dtype_fp8, int out_fp32,
                   int swiglu, int BN, int* status, int max_ctas, float act_alpha, float act_limit,
                   cudaStream_t stream);
int b200_grouped_gemm(const void* A, const void* W, void* C, const int* expert_offsets,
                      int num_experts, int total_rows, int N, int K, int lda, int ldc,
                      int dtype_fp8, int swiglu, int BN, int* status, int max_ctas, float act_alpha,
                      float act_limit, cudaStream_t stream);
int b200_moe_topk(const float* logits, const float* bias, int* topk_ids, float* topk_w, int T, int E,
                  int k, int scoring, int n_group, int topk_group, int renorm, float scale,
                  cudaStream_t stream);
int b200_argmax(const void* logits, int* out, int B, int V, long long stride, int is_fp32,
                cudaStream_t stream);
int b200_sample(const void* logits, int* out, const float* temperature, const int* top_k,
                const float* top_p, const long long* seeds, const long long* step_offset, int B,
                int V, long long stride, int is_fp32, cudaStream_t stream);
int b200_gemm_simt(const float* A, const float* W, float* C, int M, int N, int K, long long lda, long long ldw,
                   long long ldc, const int* expert_offsets, int num_experts, int act, float act_alpha,
                   float act_limit, cudaStream_t stream);
int b200_residual_norm(float* residual, long long res_stride, const int* ids, const void* table, int table_rows,
                       float table_scale, const void* a, long long a_stride, const void* b, long long b_stride,
                       const void* y, const int* slots, const float* w, int k, const void* norm_w, float eps,
                       float w_offset, void* out, long long out_stride, long long rows, int H, int n_true,
                       int is_fp32, cudaStream_t stream);
int b200_gated_rope_cache(void* q, const void* k, const void* v, void* k_cache, void* v_cache, const int* positions,
                          const int* slots, const float* cos_sin, int max_pos, int T, int Hq, int Hk, int D, int DV,
                          int DP, int DVP, int rot, int neox, long long q_stride, long long k_stride,
                          long long v_stride, int block_size, int is_fp32, cudaStream_t stream);
int b200_gated_attention(const void* q, const void* gate, const void* k_cache, const void* v_cache, void* out,
                         const int* block_tables, const int* cu_q, const int* seq_lens, int total_rows, int B,
                         int q_len, int max_q_len, int max_blocks, int block_size, int num_cache_blocks, int Hq,
                         int Hk, int D, int DV, int DP, int DVP, long long q_stride, long long g_stride,
                         long long out_stride, float scale, int window, int has_sink, float sink, int splits,
                         int is_fp32, int variant, int* status, cudaStream_t stream);
}

namespace {

// Gated activation of the GEMM epilogues (gemm/gated_act.cuh): none, silu(gate) * up, or the clamped
// form when a slope is given.
inline int act_kind(bool gated, double act_alpha) { return gated ? (act_alpha != 0.0 ? 2 : 1) : 0; }

// (BN, splits, workspace bytes, counters, cluster flag) for a problem.
std::tuple<int64_t, int64_t, int64_t, int64_t, int64_t> gemm_plan(int64_t M, int64_t N, int64_t K,
                                                                  int64_t elem_bytes, bool swiglu,
                                                                  int64_t force_bn,
                                                                  int64_t force_splits) {
  int bn, sp, cnt, cl;
  size_t ws;
  b200_gemm_plan((int)M, (int)N, (int)K, (int)elem_bytes, swiglu ? 1 : 0, (int)force_bn,
                 (int)force_splits, &bn, &sp, &ws, &cnt, &cl);
  return {bn, sp, (int64_t)ws, cnt, cl};
}

// C = A @ W^T (+bias) (+residual).  A [M,K], W [N,K]; bf16 or float8_e4m3fn.
Tensor gemm(const Tensor& a, const Tensor& w, const c10::optional<Tensor>& bias,
            const c10::optional<Tensor>& residual, bool out_fp32, bool swiglu, int64_t bn,
            int64_t splits, bool cluster_split, const c10::optional<Tensor>& workspace,
            const c10::optional<Tensor>& counters, const Tensor& status, int64_t max_ctas, double act_alpha,
            double act_limit) {
  TORCH_CHECK(a.is_cuda() && w.is_cuda() && a.dim() == 2 && w.dim() == 2, "gemm: 2-D CUDA tensors");
  TORCH_CHECK(a.scalar_type() == w.scalar_type(), "gemm: dtype mismatch");
  const bool fp8 = a.scalar_type() == at::kFloat8_e4m3fn;
  TORCH_CHECK(fp8 || a.scalar_type() == at::kBFloat16, "gemm: bf16 or float8_e4m3fn inputs");
  TORCH_CHECK(a.stride(1) == 1 && w.stride(1) == 1, "gemm: K must be contiguous");
  const int M = a.size(0), K = a.size(1), N = w.size(0);
  TORCH_CHECK(w.size(1) == K, "gemm: K mismatch");
  c10::cuda::CUDAGuard guard(a.device());
  const int n_out = swiglu ? N / 2 : N;
  Tensor c = torch::empty({M, n_out}, a.options().dtype(out_fp32 ? at::kFloat : at::kBFloat16));
  const void* bias_p = nullptr;
  const void* res_p = nullptr;
  if (bias.has_value()) {
    CHECK_CUDA_BF16(*bias);
    TORCH_CHECK(bias->numel() == N && bias->is_contiguous(), "gemm: bias [N]");
    bias_p = bias->data_ptr();
  }
  if (residual.has_value()) {
    CHECK_CUDA_BF16(*residual);
    TORCH_CHECK(residual->is_contiguous() && residual->size(0) == M && residual->size(1) == n_out,
                "gemm: residual [M,N] contiguous");
    res_p = residual->data_ptr();
  }
  void* ws_p = nullptr;
  int* cnt_p = nullptr;
  if (splits > 1 && !cluster_split) {
    TORCH_CHECK(workspace.has_value() && counters.has_value(), "gemm: split-K needs workspace");
    ws_p = workspace->data_ptr();
    cnt_p = counters->data_ptr<int>();
  }
  check(b200_gemm(a.data_ptr(), w.data_ptr(), c.data_ptr(), bias_p, res_p, M, N, K,
                  (int)a.stride(0), (int)w.stride(0), n_out, fp8 ? 1 : 0, out_fp32 ? 1 : 0,
                  act_kind(swiglu, act_alpha), (int)bn, (int)splits, cluster_split ? 1 : 0, ws_p, cnt_p,
                  status.data_ptr<int>(), (int)max_ctas, (float)act_alpha, (float)act_limit, cur_stream()),
        "gemm");
  return c;
}

// Same contract as gemm() without split-K, run by CTA pairs: one 256 x BN tile per pair of SMs
// (tcgen05 cta_group::2), each SM staging half of the weight tile.
Tensor gemm_pair(const Tensor& a, const Tensor& w, const c10::optional<Tensor>& bias,
                 const c10::optional<Tensor>& residual, bool out_fp32, bool swiglu, int64_t bn,
                 const Tensor& status, int64_t max_ctas, double act_alpha, double act_limit) {
  TORCH_CHECK(a.is_cuda() && w.is_cuda() && a.dim() == 2 && w.dim() == 2, "gemm_pair: 2-D CUDA tensors");
  TORCH_CHECK(a.scalar_type() == w.scalar_type(), "gemm_pair: dtype mismatch");
  const bool fp8 = a.scalar_type() == at::kFloat8_e4m3fn;
  TORCH_CHECK(fp8 || a.scalar_type() == at::kBFloat16, "gemm_pair: bf16 or float8_e4m3fn inputs");
  TORCH_CHECK(a.stride(1) == 1 && w.stride(1) == 1, "gemm_pair: K must be contiguous");
  const int M = a.size(0), K = a.size(1), N = w.size(0);
  TORCH_CHECK(w.size(1) == K, "gemm_pair: K mismatch");
  c10::cuda::CUDAGuard guard(a.device());
  const int n_out = swiglu ? N / 2 : N;
  Tensor c = torch::empty({M, n_out}, a.options().dtype(out_fp32 ? at::kFloat : at::kBFloat16));
  const void* bias_p = nullptr;
  const void* res_p = nullptr;
  if (bias.has_value()) {
    CHECK_CUDA_BF16(*bias);
    TORCH_CHECK(bias->numel() == N && bias->is_contiguous(), "gemm_pair: bias [N]");
    bias_p = bias->data_ptr();
  }
  if (residual.has_value()) {
    CHECK_CUDA_BF16(*residual);
    TORCH_CHECK(residual->is_contiguous() && residual->size(0) == M && residual->size(1) == n_out,
                "gemm_pair: residual [M,N] contiguous");
    res_p = residual->data_ptr();
  }
  check(b200_gemm_pair(a.data_ptr(), w.data_ptr(), c.data_ptr(), bias_p, res_p, M, N, K,
                       (int)a.stride(0), (int)w.stride(0), n_out, fp8 ? 1 : 0, out_fp32 ? 1 : 0,
                       act_kind(swiglu, act_alpha), (int)bn, status.data_ptr<int>(), (int)max_ctas,
                       (float)act_alpha, (float)act_limit, cur_stream()),
        "gemm_pair");
  return c;
}

Tensor grouped_gemm(const Tensor& a, const Tensor& w, const Tensor& expert_offsets, bool swiglu,
                    int64_t bn, const Tensor& status, int64_t max_ctas, double act_alpha, double act_limit) {
  TORCH_CHECK(a.is_cuda() && w.is_cuda() && a.dim() == 2 && w.dim() == 3, "grouped_gemm: shapes");
  TORCH_CHECK(a.scalar_type() == w.scalar_type(), "grouped_gemm: dtype mismatch");
  const bool fp8 = a.scalar_type() == at::kFloat8_e4m3fn;
  TORCH_CHECK(fp8 || a.scalar_type() == at::kBFloat16, "grouped_gemm: bf16 or fp8 inputs");
  TORCH_CHECK(a.stride(1) == 1 && w.is_contiguous(), "grouped_gemm: contiguity");
  CHECK_I32(expert_offsets);
  const int E = w.size(0), N = w.size(1), K = w.size(2), rows = a.size(0);
  TORCH_CHECK(a.size(1) == K && expert_offsets.numel() == E + 1, "grouped_gemm: size mismatch");
  c10::cuda::CUDAGuard guard(a.device());
  const int n_out = swiglu ? N / 2 : N;
  Tensor c = torch::empty({rows, n_out}, a.options().dtype(at::kBFloat16));
  check(b200_grouped_gemm(a.data_ptr(), w.data_ptr(), c.data_ptr(), expert_offsets.data_ptr<int>(),
                          E, rows, N, K, (int)a.stride(0), n_out, fp8 ? 1 : 0, act_kind(swiglu, act_alpha), (int)bn,
                          status.data_ptr<int>(), (int)max_ctas, (float)act_alpha, (float)act_limit, cur_stream()),
        "grouped_gemm");
  return c;
}

// Router: gate logits [T,E] fp32 -> (top-k ids int32 [T,k], weights fp32 [T,k]).
std::tuple<Tensor, Tensor> moe_topk(const Tensor& logits, const c10::optional<Tensor>& bias,
                                    int64_t k, bool sigmoid, int64_t n_group, int64_t topk_group,
                                    bool renorm, double scale) {
  TORCH_CHECK(logits.is_cuda() && logits.scalar_type() == at::kFloat && logits.is_contiguous() &&
                  logits.dim() == 2,
              "moe_topk: logits [T,E] fp32 contiguous");
  const int T = logits.size(0), E = logits.size(1);
  c10::cuda::CUDAGuard guard(logits.device());
  Tensor ids = torch::empty({T, k}, logits.options().dtype(at::kInt));
  Tensor w = torch::empty({T, k}, logits.options());
  const float* bp = nullptr;
  if (bias.has_value()) {
    TORCH_CHECK(bias->scalar_type() == at::kFloat && bias->numel() == E && bias->is_contiguous(),
                "moe_topk: bias [E] fp32");
    bp = bias->data_ptr<float>();
  }
  check(b200_moe_topk(logits.data_ptr<float>(), bp, ids.data_ptr<int>(), w.data_ptr<float>(), T, E,
                      (int)k, sigmoid ? 1 : 0, (int)n_group, (int)topk_group, renorm ? 1 : 0,
                      (float)scale, cur_stream()),
        "moe_topk");
  return {ids, w};
}

Tensor argmax(const Tensor& logits) {
  TORCH_CHECK(logits.is_cuda() && logits.dim() == 2 && logits.stride(1) == 1, "argmax: [B,V]");
  const bool f32 = logits.scalar_type() == at::kFloat;
  TORCH_CHECK(f32 || logits.scalar_type() == at::kBFloat16, "argmax: fp32 or bf16");
  c10::cuda::CUDAGuard guard(logits.device());
  Tensor out = torch::empty({logits.size(0)}, logits.options().dtype(at::kInt));
  check(b200_argmax(logits.data_ptr(), out.data_ptr<int>(), (int)logits.size(0),
                    (int)logits.size(1), logits.stride(0), f32 ? 1 : 0, cur_stream()),
        "argmax");
  return out;
}

Tensor sample(const Tensor& logits, const c10::optional<Tensor>& temperature,
              const c10::optional<Tensor>& top_k, const c10::optional<Tensor>& top_p,
              const c10::optional<Tensor>& seeds, const c10::optional<Tensor>& step_offset) {
  TORCH_CHECK(logits.is_cuda() && logits.dim() == 2 && logits.stride(1) == 1, "sample: [B,V]");
  const bool f32 = logits.scalar_type() == at::kFloat;
  TORCH_CHECK(f32 || logits.scalar_type() == at::kBFloat16, "sample: fp32 or bf16");
  c10::cuda::CUDAGuard guard(logits.device());
  Tensor out = torch::empty({logits.size(0)}, logits.options().dtype(at::kInt));
  check(b200_sample(logits.data_ptr(), out.data_ptr<int>(),
                    temperature.has_value() ? temperature->data_ptr<float>() : nullptr,
                    top_k.has_value() ? top_k->data_ptr<int>() : nullptr,
                    top_p.has_value() ? top_p->data_ptr<float>() : nullptr,
                    seeds.has_value() ? (const long long*)seeds->data_ptr<int64_t>() : nullptr,
                    step_offset.has_value() ? (const long long*)step_offset->data_ptr<int64_t>() : nullptr,
                    (int)logits.size(0), (int)logits.size(1), logits.stride(0), f32 ? 1 : 0,
                    cur_stream()),
        "sample");
  return out;
}

inline bool is_f32(const Tensor& t) {
  TORCH_CHECK(t.scalar_type() == at::kFloat || t.scalar_type() == at::kBFloat16, "expected bf16 or fp32");
  return t.scalar_type() == at::kFloat;
}

#define CHECK_ROWS(t, dt) \
  TORCH_CHECK((t).is_cuda() && (t).scalar_type() == (dt) && (t).dim() == 2 && (t).stride(1) == 1, #t ": 2-D rows of the call's type")

// fp32 A [M,K] @ W [N,K]^T; with expert_offsets W is [E,N,K] and rows belong to experts in order.
Tensor gemm_simt(const Tensor& a, const Tensor& w, const c10::optional<Tensor>& expert_offsets, bool swiglu,
                 double act_alpha, double act_limit) {
  CHECK_ROWS(a, at::kFloat);
  TORCH_CHECK(w.is_cuda() && w.scalar_type() == at::kFloat && w.is_contiguous(), "gemm_simt: fp32 weights");
  const bool grouped = expert_offsets.has_value();
  TORCH_CHECK(w.dim() == (grouped ? 3 : 2) && w.size(-1) == a.size(1), "gemm_simt: shapes");
  const int E = grouped ? (int)w.size(0) : 0;
  if (grouped) {
    CHECK_I32(*expert_offsets);
    TORCH_CHECK(expert_offsets->numel() == E + 1, "gemm_simt: offsets [E + 1]");
  }
  const int M = a.size(0), N = w.size(-2), K = a.size(1);
  c10::cuda::CUDAGuard guard(a.device());
  const int n_out = swiglu ? N / 2 : N;
  Tensor c = torch::empty({M, n_out}, a.options());
  check(b200_gemm_simt(a.data_ptr<float>(), w.data_ptr<float>(), c.data_ptr<float>(), M, N, K, a.stride(0), K, n_out,
                       grouped ? expert_offsets->data_ptr<int>() : nullptr, E, act_kind(swiglu, act_alpha),
                       (float)act_alpha, (float)act_limit, cur_stream()),
        "gemm_simt");
  return c;
}

// residual [T,H] fp32 is set from the table (ids given) or advanced by a + b + sum w * y[slots], then
// normalised into the returned rows (empty when there is no norm weight).
Tensor residual_norm(Tensor residual, const c10::optional<Tensor>& ids, const c10::optional<Tensor>& table,
                     double table_scale, const c10::optional<Tensor>& a, const c10::optional<Tensor>& b,
                     const c10::optional<Tensor>& y, const c10::optional<Tensor>& slots,
                     const c10::optional<Tensor>& weights, const c10::optional<Tensor>& norm_w, double eps,
                     double w_offset, int64_t n_true, bool out_fp32) {
  CHECK_ROWS(residual, at::kFloat);
  const int64_t T = residual.size(0), H = residual.size(1);
  const auto dt = out_fp32 ? at::kFloat : at::kBFloat16;
  c10::cuda::CUDAGuard guard(residual.device());
  const int* ids_p = nullptr;
  const void* table_p = nullptr;
  int table_rows = 0;
  if (ids.has_value()) {
    CHECK_I32(*ids);
    TORCH_CHECK(table.has_value() && table->is_cuda() && table->scalar_type() == dt && table->is_contiguous() &&
                    table->dim() == 2 && table->size(1) == H && table->size(0) > 0 && ids->numel() >= T,
                "residual_norm: table [rows, H]");
    ids_p = ids->data_ptr<int>();
    table_p = table->data_ptr();
    table_rows = (int)table->size(0);
  }
  const void *ap = nullptr, *bp = nullptr, *yp = nullptr;
  long long as = 0, bs = 0;
  if (a.has_value()) {
    CHECK_ROWS(*a, dt);
    TORCH_CHECK(a->size(0) == T && a->size(1) == H, "residual_norm: a [T,H]");
    ap = a->data_ptr();
    as = a->stride(0);
  }
  if (b.has_value()) {
    CHECK_ROWS(*b, dt);
    TORCH_CHECK(b->size(0) == T && b->size(1) == H, "residual_norm: b [T,H]");
    bp = b->data_ptr();
    bs = b->stride(0);
  }
  const int* sp = nullptr;
  const float* wp = nullptr;
  int k = 0;
  if (y.has_value()) {
    CHECK_ROWS(*y, dt);
    TORCH_CHECK(y->is_contiguous() && y->size(1) == H && slots.has_value() && weights.has_value(),
                "residual_norm: y [rows,H] with slots and weights");
    TORCH_CHECK(weights->is_cuda() && weights->scalar_type() == at::kFloat && weights->is_contiguous() &&
                    weights->dim() == 2 && weights->size(0) == T, "residual_norm: weights [T,k] fp32");
    CHECK_I32(*slots);
    k = (int)weights->size(1);
    TORCH_CHECK(slots->numel() >= T * k, "residual_norm: slots [T,k]");
    yp = y->data_ptr();
    sp = slots->data_ptr<int>();
    wp = weights->data_ptr<float>();
  }
  Tensor out;
  const void* nw = nullptr;
  if (norm_w.has_value()) {
    TORCH_CHECK(norm_w->is_cuda() && norm_w->scalar_type() == dt && norm_w->is_contiguous() && norm_w->numel() == H,
                "residual_norm: norm weight [H]");
    nw = norm_w->data_ptr();
    out = torch::empty({T, H}, residual.options().dtype(dt));
  } else {
    out = torch::empty({0, H}, residual.options().dtype(dt));
  }
  check(b200_residual_norm(residual.data_ptr<float>(), residual.stride(0), ids_p, table_p, table_rows,
                           (float)table_scale, ap, as, bp, bs, yp, sp, wp, k, nw, (float)eps, (float)w_offset,
                           nw ? out.data_ptr() : nullptr, H, T, (int)H, (int)n_true, out_fp32 ? 1 : 0, cur_stream()),
        "residual_norm");
  return out;
}

void check_gated_caches(const Tensor& k_cache, const Tensor& v_cache, at::ScalarType dt, int64_t head_dim,
                        int64_t head_dim_v) {
  TORCH_CHECK(k_cache.is_cuda() && v_cache.is_cuda() && k_cache.scalar_type() == dt && v_cache.scalar_type() == dt &&
                  k_cache.is_contiguous() && v_cache.is_contiguous() && k_cache.dim() == 4 && v_cache.dim() == 4,
              "gated attention: caches [blocks, Hk, block_size, D] of the call's type");
  for (int i = 0; i < 3; ++i) TORCH_CHECK(k_cache.size(i) == v_cache.size(i), "gated attention: cache shapes");
  TORCH_CHECK(k_cache.size(3) >= head_dim && v_cache.size(3) >= head_dim_v, "gated attention: cache rows too narrow");
}

void gated_rope_cache(Tensor q, const Tensor& k, const Tensor& v, Tensor k_cache, Tensor v_cache,
                      const Tensor& positions, const Tensor& slots, const Tensor& cos_sin, int64_t head_dim,
                      int64_t head_dim_v, int64_t rot, bool neox) {
  const auto dt = q.scalar_type();
  const bool f32 = is_f32(q);
  CHECK_ROWS(q, dt);
  CHECK_ROWS(k, dt);
  CHECK_ROWS(v, dt);
  CHECK_I32(positions);
  CHECK_I32(slots);
  check_gated_caches(k_cache, v_cache, dt, head_dim, head_dim_v);
  const int T = q.size(0), Hk = k_cache.size(1);
  TORCH_CHECK(positions.numel() >= T && slots.numel() >= T && q.size(1) % head_dim == 0 &&
                  k.size(0) == T && v.size(0) == T && k.size(1) == Hk * head_dim && v.size(1) == Hk * head_dim_v,
              "gated_rope_cache: shapes");
  TORCH_CHECK(cos_sin.is_cuda() && cos_sin.scalar_type() == at::kFloat && cos_sin.is_contiguous() &&
                  cos_sin.dim() == 2 && cos_sin.size(1) == rot, "gated_rope_cache: cos_sin [max_pos, rot] fp32");
  c10::cuda::CUDAGuard guard(q.device());
  check(b200_gated_rope_cache(q.data_ptr(), k.data_ptr(), v.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(),
                              positions.data_ptr<int>(), slots.data_ptr<int>(), cos_sin.data_ptr<float>(),
                              (int)cos_sin.size(0), T, (int)(q.size(1) / head_dim), Hk, (int)head_dim,
                              (int)head_dim_v, (int)k_cache.size(3), (int)v_cache.size(3), (int)rot, neox ? 1 : 0,
                              q.stride(0), k.stride(0), v.stride(0), (int)k_cache.size(2), f32 ? 1 : 0, cur_stream()),
        "gated_rope_cache");
}

// out [T, >= Hq * Dv] receives the rows (columns beyond the heads are left alone).
void gated_attention(const Tensor& q, const c10::optional<Tensor>& gate, const Tensor& k_cache, const Tensor& v_cache,
                     Tensor out, const Tensor& block_tables, const c10::optional<Tensor>& cu_q,
                     const Tensor& seq_lens, int64_t num_seqs, int64_t q_len, int64_t max_q_len, int64_t num_q_heads,
                     int64_t head_dim, int64_t head_dim_v, double scale, int64_t window, bool has_sink, double sink,
                     int64_t splits, int64_t variant, const Tensor& status) {
  const auto dt = q.scalar_type();
  const bool f32 = is_f32(q);
  CHECK_ROWS(q, dt);
  CHECK_ROWS(out, dt);
  check_gated_caches(k_cache, v_cache, dt, head_dim, head_dim_v);
  const int64_t T = q.size(0);
  TORCH_CHECK(q.size(1) == num_q_heads * head_dim && out.size(0) == T && out.size(1) >= num_q_heads * head_dim_v,
              "gated_attention: shapes");
  TORCH_CHECK(block_tables.is_cuda() && block_tables.scalar_type() == at::kInt && block_tables.dim() == 2 &&
                  block_tables.stride(1) == 1 && block_tables.size(0) >= num_seqs, "gated_attention: block tables");
  CHECK_I32(seq_lens);
  TORCH_CHECK(seq_lens.numel() >= num_seqs && num_q_heads % k_cache.size(1) == 0, "gated_attention: sequences");
  const int* cu = nullptr;
  if (cu_q.has_value()) {
    CHECK_I32(*cu_q);
    TORCH_CHECK(cu_q->numel() >= num_seqs + 1, "gated_attention: cu_q [B + 1]");
    cu = cu_q->data_ptr<int>();
  } else {
    TORCH_CHECK(T == num_seqs * q_len, "gated_attention: rows");
  }
  const void* gp = nullptr;
  long long gs = 0;
  if (gate.has_value()) {
    CHECK_ROWS(*gate, dt);
    TORCH_CHECK(gate->size(0) == T && gate->size(1) == num_q_heads * head_dim_v, "gated_attention: gate [T, Hq * Dv]");
    gp = gate->data_ptr();
    gs = gate->stride(0);
  }
  c10::cuda::CUDAGuard guard(q.device());
  check(b200_gated_attention(q.data_ptr(), gp, k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(),
                             block_tables.data_ptr<int>(), cu, seq_lens.data_ptr<int>(), (int)T, (int)num_seqs,
                             (int)q_len, (int)max_q_len, (int)block_tables.stride(0), (int)k_cache.size(2),
                             (int)k_cache.size(0), (int)num_q_heads, (int)k_cache.size(1), (int)head_dim,
                             (int)head_dim_v, (int)k_cache.size(3), (int)v_cache.size(3), q.stride(0), gs,
                             out.stride(0), (float)scale, (int)window, has_sink ? 1 : 0, (float)sink, (int)splits,
                             f32 ? 1 : 0, (int)variant, status.data_ptr<int>(), cur_stream()),
        "gated_attention");
}

}  // namespace

TORCH_LIBRARY(omni_b200, m) {
  m.def("gemm_plan", &gemm_plan);
  m.def("gemm", &gemm);
  m.def("gemm_pair", &gemm_pair);
  m.def("grouped_gemm", &grouped_gemm);
  m.def("moe_topk", &moe_topk);
  m.def("argmax", &argmax);
  m.def("sample", &sample);
  m.def("gemm_simt", &gemm_simt);
  m.def("residual_norm", &residual_norm);
  m.def("gated_rope_cache", &gated_rope_cache);
  m.def("gated_attention", &gated_attention);
}

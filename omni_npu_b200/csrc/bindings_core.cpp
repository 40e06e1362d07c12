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
int b200_gemm_simt(const float* A, const float* W, float* C, const float* bias, int M, int N, int K, long long lda, long long ldw,
                   long long ldc, const int* expert_offsets, int num_experts, int act, float act_alpha,
                   float act_limit, cudaStream_t stream);
int b200_residual_norm(float* residual, long long res_stride, const int* ids, const void* table, int table_rows,
                       float table_scale, const void* a, long long a_stride, const void* b, long long b_stride,
                       const void* y, const int* slots, const float* w, int k, float mult, const void* norm_w, float eps,
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
                         int is_fp32, int variant, int* status, int contiguous, cudaStream_t stream);
int b200_hyper_norm(const float* streams, float* streams_out, const int* ids, const void* table, int table_rows,
                    const void* y, long long y_stride, const void* ls, const float* mix, const float* w_out,
                    const float* w_in, const void* norm_w, const void* norm_b, float eps, float out_scale,
                    const void* mu, float* state, const int* seq_idx, const int* state_slots, const int* cu_q,
                    const int* seq_lens, void* out, int T, int N, int W, int n_true, int is_fp32, cudaStream_t stream);
int b200_gated_linear_prep(const void* proj, long long stride, int q_off, int f_off, int heads, int dim,
                           const float* f_bias, const float* lower, float* q, float* k, int T, int is_fp32,
                           cudaStream_t stream);
int b200_delta_prep(const void* proj, long long stride, const void* low, long long low_stride, int q_off, int k_off,
                    int v_off, int b_off, int heads, int groups, int dim, int vdim, int taps, int channels,
                    const void* conv_w, const void* conv_state, const float* dt_bias, const float* a_log,
                    float unit_eps, float q_scale, const int* seq_idx, const int* state_slots, const int* cu_q,
                    const int* seq_lens, float* q, float* k, float* g, void* v, float* beta, int T, int is_fp32,
                    cudaStream_t stream);
int b200_recurrent_scan(const float* q, const float* k, const float* g, const void* v, long long v_stride,
                        const float* beta, float* state, float* o, const int* state_slots, const int* cu_q,
                        const int* seq_lens, int B, int H, int G, int E, int DP, const void* proj,
                        long long proj_stride, void* conv_state, int keep, int channels, int mode, int is_fp32,
                        cudaStream_t stream);
int b200_head_norm_gate(const float* o, const void* w, int w_step, const void* gate, long long gate_stride,
                        int gate_silu, void* out, long long out_stride, int out_width, int T, int H, int E, float eps,
                        float scale, int is_fp32, cudaStream_t stream);
int b200_token_mix(const void* h, long long h_stride, const void* mu, int n, float* state, const int* seq_idx,
                   const int* state_slots, const int* cu_q, const int* seq_lens, void* out, int* offsets, int T, int W,
                   int is_fp32, cudaStream_t stream);
int b200_decay_prep(const void* q, long long q_stride, const void* k, long long k_stride, const float* z,
                    long long z_stride, const float* bias, const float* u, float* q_out, float* k_out, float* g_out,
                    float* bonus, int T, int heads, int dim, float q_scale, float inv_tau, int is_fp32,
                    cudaStream_t stream);
int b200_qk_norm_rope(const void* q, const void* k, const void* v, const void* v_first, void* q_out, void* k_cache,
                      void* v_cache, const int* positions, const int* slots, const float* cos_sin, int max_pos, int norm,
                      const void* q_w, const void* k_w, const float* sums, int n_q, int n_k, float eps, float lambda,
                      int T, int Hq, int Hk, int Hv, int D, int DV, int DP, int DVP, int rot, long long q_stride,
                      long long k_stride, long long v_stride, long long f_stride, int block_size, float temp, int temp_every,
                      int is_fp32, cudaStream_t stream);
int b200_latent_prep(void* q, long long q_stride, const void* kv, long long kv_stride, const void* norm_w, float eps,
                     void* cache, const int* positions, const int* slots, const float* cos_sin, int max_pos, int T,
                     int H, int dim, int rot, int rank, int row, int neox, void* q_latent, int num_latent, const void* low,
                     long long low_stride, const void* low_w, void* low_out, int low_rank, int low_width, int is_fp32,
                     cudaStream_t stream);
int b200_mixed_attention_kind(int Hs, int Hk, int Ho, int Hv, int DP, int DVP, int prompt, int is_fp32);
int b200_mixed_attention(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_tables,
                         const int* cu_q, const int* seq_lens, const float* r1, const float* r2, const float* talk,
                         const float* sink, int B, int rows, int q_len, int max_keys, int max_blocks, int block_size,
                         int Hs, int Hk, int Ho, int Hv, int D, int DV, int DP, int DVP, long long q_stride,
                         long long out_stride, float scale, float softcap, int kind, int talk_terms, int splits, float* scratch,
                         int tile0, int tiles, long long pitch, int is_fp32, cudaStream_t stream);
int b200_post_norm_residual(float* residual, long long res_stride, const int* ids, const void* table, int table_rows,
                            const void* y, long long y_stride, const void* w, int groups, const void* out_w,
                            int out_groups, void* out, long long out_stride, float eps, long long rows, int W, int n_true,
                            int is_fp32, cudaStream_t stream);
int b200_gelu_rows(const void* z, long long z_stride, const int* ids, const void* table, int table_rows,
                   long long table_stride, int offset, int dim, int width, void* out, int T, int is_fp32,
                   cudaStream_t stream);
int b200_head_gemm(const void* a, long long a_t, long long a_h, const void* w, void* out, long long o_t, long long o_h,
                   int T, int H, int N, int K, int is_fp32, cudaStream_t stream);
int b200_latent_gather(const void* cache, void* out, const int* block_tables, const int* seq_lens, const int* start,
                       int B, int max_len, int max_blocks, int block_size, int row_bytes, int total,
                       cudaStream_t stream);
size_t b200_latent_decode_scratch_bytes(int total_tokens, int N, int rank, int splits);
int b200_latent_decode(const void* q, const void* cache, void* out, const int* block_tables, const int* seq_lens, int B,
                       int N, int row, int rank, int max_blocks, int block_size, int num_cache_blocks, float scale,
                       int splits, void* scratch, int* status, cudaStream_t stream);
}

namespace {

// Activation kinds of the GEMM epilogues are those of gemm/gated_act.cuh; 1, 2, 4 and 7 join pairs of columns.
inline bool gated(int64_t act) { return act == 1 || act == 2 || act == 4 || act == 7; }

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
            const c10::optional<Tensor>& residual, bool out_fp32, int64_t act, int64_t bn,
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
  const int n_out = gated(act) ? N / 2 : N;
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
                  (int)act, (int)bn, (int)splits, cluster_split ? 1 : 0, ws_p, cnt_p,
                  status.data_ptr<int>(), (int)max_ctas, (float)act_alpha, (float)act_limit, cur_stream()),
        "gemm");
  return c;
}

// Same contract as gemm() without split-K, run by CTA pairs: one 256 x BN tile per pair of SMs
// (tcgen05 cta_group::2), each SM staging half of the weight tile.
Tensor gemm_pair(const Tensor& a, const Tensor& w, const c10::optional<Tensor>& bias,
                 const c10::optional<Tensor>& residual, bool out_fp32, int64_t act, int64_t bn,
                 const Tensor& status, int64_t max_ctas, double act_alpha, double act_limit) {
  TORCH_CHECK(a.is_cuda() && w.is_cuda() && a.dim() == 2 && w.dim() == 2, "gemm_pair: 2-D CUDA tensors");
  TORCH_CHECK(a.scalar_type() == w.scalar_type(), "gemm_pair: dtype mismatch");
  const bool fp8 = a.scalar_type() == at::kFloat8_e4m3fn;
  TORCH_CHECK(fp8 || a.scalar_type() == at::kBFloat16, "gemm_pair: bf16 or float8_e4m3fn inputs");
  TORCH_CHECK(a.stride(1) == 1 && w.stride(1) == 1, "gemm_pair: K must be contiguous");
  const int M = a.size(0), K = a.size(1), N = w.size(0);
  TORCH_CHECK(w.size(1) == K, "gemm_pair: K mismatch");
  c10::cuda::CUDAGuard guard(a.device());
  const int n_out = gated(act) ? N / 2 : N;
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
                       (int)act, (int)bn, status.data_ptr<int>(), (int)max_ctas,
                       (float)act_alpha, (float)act_limit, cur_stream()),
        "gemm_pair");
  return c;
}

Tensor grouped_gemm(const Tensor& a, const Tensor& w, const Tensor& expert_offsets, int64_t act,
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
  const int n_out = gated(act) ? N / 2 : N;
  Tensor c = torch::empty({rows, n_out}, a.options().dtype(at::kBFloat16));
  check(b200_grouped_gemm(a.data_ptr(), w.data_ptr(), c.data_ptr(), expert_offsets.data_ptr<int>(),
                          E, rows, N, K, (int)a.stride(0), n_out, fp8 ? 1 : 0, (int)act, (int)bn,
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
Tensor gemm_simt(const Tensor& a, const Tensor& w, const c10::optional<Tensor>& expert_offsets, int64_t act,
                 double act_alpha, double act_limit, const c10::optional<Tensor>& bias) {
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
  const float* bias_p = nullptr;
  if (bias.has_value()) {
    TORCH_CHECK(bias->is_cuda() && bias->scalar_type() == at::kFloat && bias->is_contiguous() && bias->numel() == N,
                "gemm_simt: bias [N] fp32");
    bias_p = bias->data_ptr<float>();
  }
  c10::cuda::CUDAGuard guard(a.device());
  const int n_out = gated(act) ? N / 2 : N;
  Tensor c = torch::empty({M, n_out}, a.options());
  check(b200_gemm_simt(a.data_ptr<float>(), w.data_ptr<float>(), c.data_ptr<float>(), bias_p, M, N, K, a.stride(0), K, n_out,
                       grouped ? expert_offsets->data_ptr<int>() : nullptr, E, (int)act,
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
                     double w_offset, int64_t n_true, bool out_fp32, double mult) {
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
                           (float)table_scale, ap, as, bp, bs, yp, sp, wp, k, (float)mult, nw, (float)eps, (float)w_offset,
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
                     int64_t splits, int64_t variant, const Tensor& status, bool contiguous) {
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
                             f32 ? 1 : 0, (int)variant, status.data_ptr<int>(), contiguous ? 1 : 0, cur_stream()),
        "gated_attention");
}

#define CHECK_F32(t) TORCH_CHECK((t).is_cuda() && (t).scalar_type() == at::kFloat && (t).is_contiguous(), #t ": contiguous fp32")
#define CHECK_VEC(t, dt, n) \
  TORCH_CHECK((t).is_cuda() && (t).scalar_type() == (dt) && (t).is_contiguous() && (t).numel() == (n), #t ": vector of the call's type and width")

// Joins y to the streams (or starts them from the table), reads and normalises: (streams, rows).
std::tuple<Tensor, Tensor> hyper_norm(const c10::optional<Tensor>& streams, const c10::optional<Tensor>& ids,
                                      const c10::optional<Tensor>& table, int64_t N, const c10::optional<Tensor>& y,
                                      const c10::optional<Tensor>& ls, const c10::optional<Tensor>& mix,
                                      const c10::optional<Tensor>& w_out, const Tensor& w_in, const Tensor& norm_w,
                                      const Tensor& norm_b, double eps, int64_t n_true, double out_scale,
                                      const c10::optional<Tensor>& mu, const c10::optional<Tensor>& state,
                                      const c10::optional<Tensor>& seq_idx, const c10::optional<Tensor>& state_slots,
                                      const c10::optional<Tensor>& cu_q, const c10::optional<Tensor>& seq_lens,
                                      bool keep) {
  const auto dt = norm_w.scalar_type();
  const bool f32 = is_f32(norm_w);
  const int64_t W = norm_w.numel();
  CHECK_VEC(norm_w, dt, W);
  CHECK_VEC(norm_b, dt, W);
  CHECK_F32(w_in);
  TORCH_CHECK(w_in.numel() == N && N >= 1 && N <= 8, "hyper_norm: 1 to 8 streams");
  c10::cuda::CUDAGuard guard(norm_w.device());
  int64_t T;
  const float *x = nullptr, *mix_p = nullptr, *out_p = nullptr;
  const int* ids_p = nullptr;
  const void *table_p = nullptr, *y_p = nullptr, *ls_p = nullptr;
  int table_rows = 0;
  long long ys = 0;
  if (ids.has_value()) {
    CHECK_I32(*ids);
    TORCH_CHECK(table.has_value() && table->is_cuda() && table->scalar_type() == dt && table->is_contiguous() &&
                    table->dim() == 2 && table->size(1) == W && table->size(0) > 0, "hyper_norm: table [rows, W]");
    T = ids->numel();
    ids_p = ids->data_ptr<int>();
    table_p = table->data_ptr();
    table_rows = (int)table->size(0);
  } else {
    TORCH_CHECK(streams.has_value() && y.has_value() && ls.has_value() && mix.has_value() && w_out.has_value(),
                "hyper_norm: streams with a sublayer's result");
    CHECK_F32(*streams);
    CHECK_F32(*mix);
    CHECK_F32(*w_out);
    CHECK_ROWS(*y, dt);
    CHECK_VEC(*ls, dt, W);
    T = streams->size(0);
    TORCH_CHECK(streams->dim() == 3 && streams->size(1) == N && streams->size(2) == W && y->size(0) == T &&
                    y->size(1) == W && mix->numel() == N * N && w_out->numel() == N, "hyper_norm: shapes");
    x = streams->data_ptr<float>();
    y_p = y->data_ptr();
    ys = y->stride(0);
    ls_p = ls->data_ptr();
    mix_p = mix->data_ptr<float>();
    out_p = w_out->data_ptr<float>();
  }
  const void* mu_p = nullptr;
  float* st = nullptr;
  const int *si = nullptr, *ss = nullptr, *cu = nullptr, *sl = nullptr;
  if (mu.has_value()) {
    TORCH_CHECK(state.has_value() && seq_idx.has_value() && state_slots.has_value() && cu_q.has_value() &&
                    seq_lens.has_value(), "hyper_norm: token shift arguments");
    CHECK_VEC(*mu, dt, W);
    CHECK_F32(*state);
    CHECK_I32(*seq_idx);
    CHECK_I32(*state_slots);
    CHECK_I32(*cu_q);
    CHECK_I32(*seq_lens);
    TORCH_CHECK(state->dim() == 2 && state->size(1) == W && seq_idx->numel() >= T, "hyper_norm: state [slots, W]");
    mu_p = mu->data_ptr();
    st = state->data_ptr<float>();
    si = seq_idx->data_ptr<int>();
    ss = state_slots->data_ptr<int>();
    cu = cu_q->data_ptr<int>();
    sl = seq_lens->data_ptr<int>();
  }
  Tensor out = torch::empty({T, W}, norm_w.options());
  Tensor next = torch::empty(keep ? std::vector<int64_t>{T, N, W} : std::vector<int64_t>{0}, w_in.options());
  check(b200_hyper_norm(x, keep ? next.data_ptr<float>() : nullptr, ids_p, table_p, table_rows, y_p, ys, ls_p, mix_p,
                        out_p, w_in.data_ptr<float>(), norm_w.data_ptr(), norm_b.data_ptr(), (float)eps,
                        (float)out_scale, mu_p, st, si, ss, cu, sl, out.data_ptr(), (int)T, (int)N, (int)W, (int)n_true,
                        f32 ? 1 : 0, cur_stream()),
        "hyper_norm");
  return {next, out};
}

std::tuple<Tensor, Tensor> gated_linear_prep(const Tensor& proj, int64_t q_off, int64_t f_off, int64_t heads,
                                             int64_t dim, const Tensor& f_bias, const Tensor& lower) {
  const bool f32 = is_f32(proj);
  CHECK_ROWS(proj, proj.scalar_type());
  CHECK_F32(f_bias);
  CHECK_F32(lower);
  const int64_t T = proj.size(0), n = heads * dim;
  TORCH_CHECK(f_bias.numel() == n && lower.numel() == n && q_off >= 0 && f_off >= 0 && q_off + n <= proj.size(1) &&
                  f_off + n <= proj.size(1), "gated_linear_prep: shapes");
  c10::cuda::CUDAGuard guard(proj.device());
  Tensor q = torch::empty({T, heads, (dim + 3) / 4 * 4}, f_bias.options()), k = torch::empty_like(q);
  check(b200_gated_linear_prep(proj.data_ptr(), proj.stride(0), (int)q_off, (int)f_off, (int)heads, (int)dim,
                               f_bias.data_ptr<float>(), lower.data_ptr<float>(), q.data_ptr<float>(),
                               k.data_ptr<float>(), (int)T, f32 ? 1 : 0, cur_stream()),
        "gated_linear_prep");
  return {q, k};
}

std::tuple<Tensor, Tensor, Tensor, Tensor, Tensor> delta_prep(
    const Tensor& proj, const Tensor& low, int64_t q_off, int64_t k_off, int64_t v_off, int64_t b_off, int64_t heads,
    int64_t groups, int64_t dim, int64_t vdim, const Tensor& conv_w, const Tensor& conv_state, const Tensor& dt_bias,
    const Tensor& a_log, double unit_eps, const Tensor& seq_idx, const Tensor& state_slots, const Tensor& cu_q,
    const Tensor& seq_lens) {
  const auto dt = proj.scalar_type();
  const bool f32 = is_f32(proj);
  CHECK_ROWS(proj, dt);
  CHECK_ROWS(low, dt);
  CHECK_F32(dt_bias);
  CHECK_F32(a_log);
  CHECK_I32(seq_idx);
  CHECK_I32(state_slots);
  CHECK_I32(cu_q);
  CHECK_I32(seq_lens);
  const int64_t T = proj.size(0), channels = conv_w.size(0), taps = conv_w.size(1);
  TORCH_CHECK(conv_w.is_cuda() && conv_w.scalar_type() == dt && conv_w.is_contiguous() && conv_state.is_cuda() &&
                  conv_state.scalar_type() == dt && conv_state.is_contiguous() && conv_state.dim() == 3 &&
                  conv_state.size(1) == taps - 1 && conv_state.size(2) == channels, "delta_prep: convolution");
  TORCH_CHECK(low.size(0) == T && low.size(1) == heads * dim && dt_bias.numel() == heads * dim &&
                  a_log.numel() == heads && seq_idx.numel() >= T && b_off + heads <= proj.size(1) &&
                  channels <= proj.size(1) && q_off + groups * dim <= channels && k_off + groups * dim <= channels &&
                  v_off + heads * vdim <= channels && heads % groups == 0, "delta_prep: shapes");
  c10::cuda::CUDAGuard guard(proj.device());
  const int64_t DP = (dim + 3) / 4 * 4;
  Tensor q = torch::empty({T, groups, DP}, dt_bias.options()), k = torch::empty_like(q);
  Tensor g = torch::empty({T, heads, DP}, dt_bias.options()), beta = torch::empty({T, heads}, dt_bias.options());
  Tensor v = torch::empty({T, heads * vdim}, proj.options());
  check(b200_delta_prep(proj.data_ptr(), proj.stride(0), low.data_ptr(), low.stride(0), (int)q_off, (int)k_off,
                        (int)v_off, (int)b_off, (int)heads, (int)groups, (int)dim, (int)vdim, (int)taps, (int)channels,
                        conv_w.data_ptr(), conv_state.data_ptr(), dt_bias.data_ptr<float>(), a_log.data_ptr<float>(),
                        (float)unit_eps, 1.f / sqrtf((float)dim), seq_idx.data_ptr<int>(), state_slots.data_ptr<int>(),
                        cu_q.data_ptr<int>(), seq_lens.data_ptr<int>(), q.data_ptr<float>(), k.data_ptr<float>(),
                        g.data_ptr<float>(), v.data_ptr(), beta.data_ptr<float>(), (int)T, f32 ? 1 : 0, cur_stream()),
        "delta_prep");
  return {q, k, g, v, beta};
}

Tensor recurrent_scan(const Tensor& q, const Tensor& k, const c10::optional<Tensor>& g, const Tensor& v,
                      const c10::optional<Tensor>& beta, Tensor state, int64_t heads, int64_t vdim,
                      const Tensor& state_slots, const Tensor& cu_q, const Tensor& seq_lens, int64_t num_seqs,
                      const c10::optional<Tensor>& proj, const c10::optional<Tensor>& conv_state, bool bonus) {
  CHECK_F32(q);
  CHECK_F32(k);
  CHECK_F32(state);
  CHECK_ROWS(v, v.scalar_type());
  CHECK_I32(state_slots);
  CHECK_I32(cu_q);
  CHECK_I32(seq_lens);
  const bool f32 = is_f32(v);
  TORCH_CHECK(q.dim() == 3 && q.sizes() == k.sizes(), "recurrent_scan: q, k [T, G, d]");
  const int64_t T = q.size(0), G = q.size(1), DP = q.size(2);
  TORCH_CHECK(v.size(0) == T && v.size(1) == heads * vdim && state.dim() == 4 && state.size(1) == heads &&
                  state.size(2) == vdim && state.size(3) == DP && heads % G == 0 && state_slots.numel() >= num_seqs &&
                  cu_q.numel() >= num_seqs + 1 && seq_lens.numel() >= num_seqs, "recurrent_scan: shapes");
  TORCH_CHECK(g.has_value() || !beta.has_value(), "recurrent_scan: beta without decays");
  TORCH_CHECK(!bonus || beta.has_value(), "recurrent_scan: the bonus comes in beta");
  if (g.has_value()) {
    CHECK_F32(*g);
    TORCH_CHECK(g->numel() == T * heads * DP, "recurrent_scan: g [T, H, d]");
  }
  if (beta.has_value()) {
    CHECK_F32(*beta);
    TORCH_CHECK(beta->numel() == T * heads, "recurrent_scan: beta [T, H]");
  }
  const int mode = !g.has_value() ? 0 : !beta.has_value() ? 2 : bonus ? 3 : 1;
  const void* proj_p = nullptr;
  void* cs = nullptr;
  long long ps = 0;
  int keep = 0, channels = 0;
  if (proj.has_value() && conv_state.has_value()) {
    CHECK_ROWS(*proj, v.scalar_type());
    TORCH_CHECK(conv_state->is_cuda() && conv_state->scalar_type() == v.scalar_type() && conv_state->is_contiguous() &&
                    conv_state->dim() == 3 && conv_state->size(0) == state.size(0) &&
                    conv_state->size(2) <= proj->size(1) && proj->size(0) == T, "recurrent_scan: convolution inputs");
    proj_p = proj->data_ptr();
    ps = proj->stride(0);
    cs = conv_state->data_ptr();
    keep = (int)conv_state->size(1);
    channels = (int)conv_state->size(2);
  }
  c10::cuda::CUDAGuard guard(q.device());
  Tensor o = torch::empty({T, heads, vdim}, q.options());
  check(b200_recurrent_scan(q.data_ptr<float>(), k.data_ptr<float>(), g.has_value() ? g->data_ptr<float>() : nullptr,
                            v.data_ptr(), v.stride(0), beta.has_value() ? beta->data_ptr<float>() : nullptr,
                            state.data_ptr<float>(), o.data_ptr<float>(), state_slots.data_ptr<int>(),
                            cu_q.data_ptr<int>(), seq_lens.data_ptr<int>(), (int)num_seqs, (int)heads, (int)G,
                            (int)vdim, (int)DP, proj_p, ps, cs, keep, channels, mode, f32 ? 1 : 0, cur_stream()),
        "recurrent_scan");
  return o;
}

// weight [E] for all heads or [H, E]; out (rows [T, >= H * E], any pitch) is written when given
Tensor head_norm_gate(const Tensor& o, const Tensor& weight, double eps, const c10::optional<Tensor>& gate,
                      int64_t out_width, bool gate_silu, double scale, const c10::optional<Tensor>& out_rows) {
  CHECK_F32(o);
  const auto dt = weight.scalar_type();
  const bool f32 = is_f32(weight);
  TORCH_CHECK(o.dim() == 3, "head_norm_gate: o [T, H, E]");
  const bool per_head = weight.dim() == 2;
  CHECK_VEC(weight, dt, per_head ? o.size(1) * o.size(2) : o.size(2));
  const void* gp = nullptr;
  long long gs = 0;
  if (gate.has_value()) {
    CHECK_ROWS(*gate, dt);
    TORCH_CHECK(gate->size(0) == o.size(0) && gate->size(1) == o.size(1) * o.size(2), "head_norm_gate: gate");
    gp = gate->data_ptr();
    gs = gate->stride(0);
  }
  c10::cuda::CUDAGuard guard(o.device());
  Tensor out = out_rows.has_value() ? *out_rows : torch::empty({o.size(0), out_width}, weight.options());
  CHECK_ROWS(out, dt);
  TORCH_CHECK(out.size(0) == o.size(0) && out.size(1) >= o.size(1) * o.size(2), "head_norm_gate: out [T, >= H * E]");
  check(b200_head_norm_gate(o.data_ptr<float>(), weight.data_ptr(), per_head ? (int)o.size(2) : 0, gp, gs,
                            gate_silu ? 1 : 0, out.data_ptr(), out.stride(0), (int)out.size(1), (int)o.size(0),
                            (int)o.size(1), (int)o.size(2), (float)eps, (float)scale, f32 ? 1 : 0, cur_stream()),
        "head_norm_gate");
  return out;
}

// Rows h_t + (h_(t-1) - h_t) mu_s, one blend after another: (rows [n * T, W], offsets [n + 1]).
std::tuple<Tensor, Tensor> token_mix(const Tensor& h, const Tensor& mu, Tensor state, const Tensor& seq_idx,
                                     const Tensor& state_slots, const Tensor& cu_q, const Tensor& seq_lens) {
  const auto dt = h.scalar_type();
  const bool f32 = is_f32(h);
  CHECK_ROWS(h, dt);
  CHECK_F32(state);
  CHECK_I32(seq_idx);
  CHECK_I32(state_slots);
  CHECK_I32(cu_q);
  CHECK_I32(seq_lens);
  const int64_t T = h.size(0), W = h.size(1), n = mu.size(0);
  TORCH_CHECK(mu.is_cuda() && mu.scalar_type() == dt && mu.is_contiguous() && mu.dim() == 2 && mu.size(1) == W &&
                  state.dim() == 2 && state.size(1) == W && seq_idx.numel() >= T, "token_mix: shapes");
  c10::cuda::CUDAGuard guard(h.device());
  Tensor out = torch::empty({n * T, W}, h.options()), offsets = torch::empty({n + 1}, cu_q.options());
  check(b200_token_mix(h.data_ptr(), h.stride(0), mu.data_ptr(), (int)n, state.data_ptr<float>(),
                       seq_idx.data_ptr<int>(), state_slots.data_ptr<int>(), cu_q.data_ptr<int>(),
                       seq_lens.data_ptr<int>(), out.data_ptr(), offsets.data_ptr<int>(), (int)T, (int)W, f32 ? 1 : 0,
                       cur_stream()),
        "token_mix");
  return {out, offsets};
}

// u given: time mixing (q, k, decays, bonus); else (q * q_scale, k, decays, empty).
std::tuple<Tensor, Tensor, Tensor, Tensor> decay_prep(const Tensor& q, const Tensor& k, const Tensor& z,
                                                      const Tensor& bias, const c10::optional<Tensor>& u, int64_t heads,
                                                      int64_t dim, double q_scale, double inv_tau) {
  const auto dt = q.scalar_type();
  const bool f32 = is_f32(q);
  CHECK_ROWS(q, dt);
  CHECK_ROWS(k, dt);
  CHECK_ROWS(z, at::kFloat);
  CHECK_F32(bias);
  const int64_t T = q.size(0), n = heads * dim, DP = (dim + 3) / 4 * 4;
  TORCH_CHECK(q.size(1) >= n && k.size(0) == T && k.size(1) >= n && z.size(0) == T && z.size(1) >= n &&
                  bias.numel() == n, "decay_prep: shapes");
  if (u.has_value()) {
    CHECK_F32(*u);
    TORCH_CHECK(u->numel() == n, "decay_prep: u [heads, dim]");
  }
  c10::cuda::CUDAGuard guard(q.device());
  Tensor qo = torch::empty({T, heads, DP}, bias.options()), ko = torch::empty_like(qo), go = torch::empty_like(qo);
  Tensor bonus = torch::empty({u.has_value() ? T : 0, heads}, bias.options());
  check(b200_decay_prep(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), z.data_ptr<float>(), z.stride(0),
                        bias.data_ptr<float>(), u.has_value() ? u->data_ptr<float>() : nullptr, qo.data_ptr<float>(),
                        ko.data_ptr<float>(), go.data_ptr<float>(), bonus.data_ptr<float>(), (int)T, (int)heads,
                        (int)dim, (float)q_scale, (float)inv_tau, f32 ? 1 : 0, cur_stream()),
        "decay_prep");
  return {qo, ko, go, bonus};
}

// norm: 0 none, 1 over the whole projections (weights; sums of squares [T, 2] over n_q / n_k elements when they
// were taken elsewhere), 2 per head.  Returns the queries [T, Hq * D].
Tensor qk_norm_rope(const Tensor& q, const Tensor& k, const Tensor& v, const c10::optional<Tensor>& v_first,
                    double lambda, Tensor k_cache, Tensor v_cache, const Tensor& positions, const Tensor& slots,
                    const c10::optional<Tensor>& cos_sin, int64_t head_dim, int64_t head_dim_v, int64_t rot, int64_t norm,
                    const c10::optional<Tensor>& q_w, const c10::optional<Tensor>& k_w,
                    const c10::optional<Tensor>& sums, int64_t n_q, int64_t n_k, double eps,
                    double temp, int64_t temp_every) {
  const auto dt = q.scalar_type();
  const bool f32 = is_f32(q);
  CHECK_ROWS(q, dt);
  CHECK_ROWS(k, dt);
  CHECK_ROWS(v, dt);
  CHECK_I32(positions);
  CHECK_I32(slots);
  for (const Tensor& c : {k_cache, v_cache})
    TORCH_CHECK(c.is_cuda() && c.scalar_type() == dt && c.dim() == 4 && c.is_contiguous() &&
                    c.size(0) == k_cache.size(0) && c.size(2) == k_cache.size(2),
                "qk_norm_rope: caches [blocks, heads, block_size, width]");
  TORCH_CHECK(k_cache.size(3) >= head_dim && v_cache.size(3) >= head_dim_v, "qk_norm_rope: width of the cache rows");
  const int T = q.size(0), Hk = k_cache.size(1), Hv = v_cache.size(1);
  TORCH_CHECK(positions.numel() >= T && slots.numel() >= T && q.size(1) % head_dim == 0 && k.size(0) == T &&
                  v.size(0) == T && k.size(1) == Hk * head_dim && v.size(1) == Hv * head_dim_v, "qk_norm_rope: shapes");
  const float* cs = nullptr;
  int max_pos = 1 << 30;
  if (cos_sin.has_value()) {
    TORCH_CHECK(cos_sin->is_cuda() && cos_sin->scalar_type() == at::kFloat && cos_sin->is_contiguous() &&
                    cos_sin->dim() == 2 && cos_sin->size(1) == rot, "qk_norm_rope: cos_sin [max_pos, rot] fp32");
    cs = cos_sin->data_ptr<float>();
    max_pos = (int)cos_sin->size(0);
  }
  TORCH_CHECK(cs || rot == 0, "qk_norm_rope: a rotation needs cos_sin");
  const void *qw = nullptr, *kw = nullptr, *vf = nullptr;
  const float* sp = nullptr;
  long long fs = 0;
  if (norm == 1 || norm == 3) {
    TORCH_CHECK(q_w.has_value() && k_w.has_value(), "qk_norm_rope: norm weights");
    CHECK_VEC(*q_w, dt, norm == 1 ? q.size(1) : head_dim);
    CHECK_VEC(*k_w, dt, norm == 1 ? k.size(1) : head_dim);
    qw = q_w->data_ptr();
    kw = k_w->data_ptr();
    if (norm == 1 && sums.has_value()) {
      CHECK_F32(*sums);
      TORCH_CHECK(sums->numel() == 2 * T, "qk_norm_rope: sums [T, 2]");
      sp = sums->data_ptr<float>();
    }
  }
  if (v_first.has_value()) {
    CHECK_ROWS(*v_first, dt);
    TORCH_CHECK(v_first->size(0) == T && v_first->size(1) == v.size(1), "qk_norm_rope: v_first like v");
    vf = v_first->data_ptr();
    fs = v_first->stride(0);
  }
  c10::cuda::CUDAGuard guard(q.device());
  Tensor out = torch::empty({T, q.size(1)}, q.options());
  check(b200_qk_norm_rope(q.data_ptr(), k.data_ptr(), v.data_ptr(), vf, out.data_ptr(), k_cache.data_ptr(),
                          v_cache.data_ptr(), positions.data_ptr<int>(), slots.data_ptr<int>(), cs, max_pos, (int)norm, qw, kw, sp, (int)n_q, (int)n_k, (float)eps, (float)lambda, T,
                          (int)(q.size(1) / head_dim), Hk, Hv, (int)head_dim, (int)head_dim_v, (int)k_cache.size(3),
                          (int)v_cache.size(3), (int)rot, q.stride(0), k.stride(0), v.stride(0), fs,
                          (int)k_cache.size(2), (float)temp, (int)temp_every, f32 ? 1 : 0, cur_stream()),
        "qk_norm_rope");
  return out;
}

void latent_prep(const c10::optional<Tensor>& q, const c10::optional<Tensor>& kv, const c10::optional<Tensor>& norm_w,
                 double eps, Tensor cache, const Tensor& positions, const Tensor& slots, const Tensor& cos_sin,
                 int64_t heads, int64_t dim, int64_t rot, int64_t rank, bool neox, const c10::optional<Tensor>& q_latent,
                 int64_t num_latent, const c10::optional<Tensor>& low, const c10::optional<Tensor>& low_w,
                 const c10::optional<Tensor>& low_out) {
  const auto dt = cache.scalar_type();
  const bool f32 = is_f32(cache);
  CHECK_I32(positions);
  CHECK_I32(slots);
  TORCH_CHECK(q.has_value() || kv.has_value() || low.has_value(), "latent_prep: nothing to do");
  const int64_t T = q.has_value() ? q->size(0) : kv.has_value() ? kv->size(0) : low->size(0);
  TORCH_CHECK(cache.is_cuda() && cache.is_contiguous() && cache.dim() == 3 && cache.size(2) >= rank + rot,
              "latent_prep: cache [blocks, block_size, row]");
  TORCH_CHECK(positions.numel() >= T && slots.numel() >= T, "latent_prep: positions, slots [T]");
  TORCH_CHECK(cos_sin.is_cuda() && cos_sin.scalar_type() == at::kFloat && cos_sin.is_contiguous() &&
                  cos_sin.dim() == 2 && cos_sin.size(1) == rot, "latent_prep: cos_sin [max_pos, rot] fp32");
  void *qp = nullptr, *ql = nullptr, *lo = nullptr;
  const void *kvp = nullptr, *nw = nullptr, *lp = nullptr, *lw = nullptr;
  long long qs = 0, kvs = 0, ls = 0;
  int low_rank = 0, low_width = 0;
  if (q.has_value()) {
    CHECK_ROWS(*q, dt);
    TORCH_CHECK(q->size(1) >= heads * (dim + rot), "latent_prep: q [T, heads * (dim + rot)]");
    qp = q->data_ptr();
    qs = q->stride(0);
  }
  if (kv.has_value()) {
    CHECK_ROWS(*kv, dt);
    TORCH_CHECK(kv->size(0) == T && kv->size(1) >= rank + rot && norm_w.has_value(), "latent_prep: kv [T, rank + rot]");
    CHECK_VEC(*norm_w, dt, rank);
    kvp = kv->data_ptr();
    nw = norm_w->data_ptr();
    kvs = kv->stride(0);
  }
  if (low.has_value()) {
    CHECK_ROWS(*low, dt);
    TORCH_CHECK(low_w.has_value() && low_out.has_value(), "latent_prep: weight and result of the queries' latent");
    low_rank = (int)low_w->numel();
    CHECK_VEC(*low_w, dt, low_rank);
    TORCH_CHECK(low_out->is_cuda() && low_out->scalar_type() == dt && low_out->is_contiguous() && low_out->dim() == 2 &&
                    low_out->size(0) == T && low_out->size(1) >= low_rank && low->size(0) == T &&
                    low->size(1) >= low_rank, "latent_prep: queries' latent [T, n]");
    low_width = (int)low_out->size(1);
    lp = low->data_ptr();
    lw = low_w->data_ptr();
    lo = low_out->data_ptr();
    ls = low->stride(0);
  }
  if (num_latent > 0 && q.has_value()) {
    TORCH_CHECK(q_latent.has_value() && q_latent->is_cuda() && q_latent->scalar_type() == dt &&
                    q_latent->is_contiguous() && q_latent->dim() == 3 && q_latent->size(0) >= num_latent &&
                    q_latent->size(1) == heads && q_latent->size(2) == cache.size(2), "latent_prep: q_latent");
    ql = q_latent->data_ptr();
  } else {
    num_latent = 0;
  }
  c10::cuda::CUDAGuard guard(cache.device());
  check(b200_latent_prep(qp, qs, kvp, kvs, nw, (float)eps, cache.data_ptr(), positions.data_ptr<int>(),
                         slots.data_ptr<int>(), cos_sin.data_ptr<float>(), (int)cos_sin.size(0), (int)T, (int)heads,
                         (int)dim, (int)rot, (int)rank, (int)cache.size(2), neox ? 1 : 0, ql, (int)num_latent, lp, ls, lw,
                         lo, low_rank, low_width, f32 ? 1 : 0, cur_stream()),
        "latent_prep");
}

// 0: the plain kernel, 1: the tensor-core kernels; variant 2 asks for the plain one, 1 for an error instead of it
int64_t mixed_attention_kind(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, const Tensor& talk, bool prompt,
                             int64_t variant) {
  TORCH_CHECK(k_cache.dim() == 4 && v_cache.dim() == 4 && talk.dim() == 2, "mixed_attention: shapes");
  const int kind = variant == 2 ? 0
                                : b200_mixed_attention_kind((int)talk.size(1), (int)k_cache.size(1), (int)talk.size(0),
                                                            (int)v_cache.size(1), (int)k_cache.size(3),
                                                            (int)v_cache.size(3), prompt ? 1 : 0, is_f32(q) ? 1 : 0);
  TORCH_CHECK(kind || variant != 1, "mixed_attention: these sizes are beyond the tensor-core kernels");
  return kind;
}

// out [T, >= Ho * Dv].  kind 1: `scratch` holds the partial results of split decode rows, or the mixed scores of the
// query tiles tile0 .. tile0 + tiles - 1, numbered through all portions.
void mixed_attention(const Tensor& q, const Tensor& k_cache, const Tensor& v_cache, Tensor out, const Tensor& block_tables,
                     const c10::optional<Tensor>& cu_q, const Tensor& seq_lens, int64_t num_seqs, int64_t q_len,
                     int64_t max_keys, int64_t head_dim, int64_t head_dim_v, double scale, double softcap,
                     const c10::optional<Tensor>& r1, const c10::optional<Tensor>& r2, const Tensor& talk,
                     const c10::optional<Tensor>& sink, int64_t kind, int64_t talk_terms, int64_t splits,
                     const c10::optional<Tensor>& scratch, int64_t tile0, int64_t tiles) {
  const auto dt = q.scalar_type();
  const bool f32 = is_f32(q);
  CHECK_ROWS(q, dt);
  CHECK_ROWS(out, dt);
  for (const Tensor& c : {k_cache, v_cache})
    TORCH_CHECK(c.is_cuda() && c.scalar_type() == dt && c.dim() == 4 && c.is_contiguous() &&
                    c.size(0) == k_cache.size(0) && c.size(2) == k_cache.size(2),
                "mixed_attention: caches [blocks, heads, block_size, width]");
  const int64_t T = q.size(0), Hs = talk.size(1), Ho = talk.size(0);
  TORCH_CHECK(k_cache.size(3) >= head_dim && v_cache.size(3) >= head_dim_v && q.size(1) == Hs * head_dim &&
                  out.size(0) == T && out.size(1) >= Ho * head_dim_v, "mixed_attention: shapes");
  TORCH_CHECK(block_tables.is_cuda() && block_tables.scalar_type() == at::kInt && block_tables.dim() == 2 &&
                  block_tables.stride(1) == 1 && block_tables.size(0) >= num_seqs, "mixed_attention: block tables");
  CHECK_I32(seq_lens);
  TORCH_CHECK(seq_lens.numel() >= num_seqs, "mixed_attention: sequences");
  const auto vec = [&](const c10::optional<Tensor>& t, int64_t n) -> const float* {
    if (!t.has_value()) return nullptr;
    TORCH_CHECK(t->is_cuda() && t->scalar_type() == at::kFloat && t->is_contiguous() && t->numel() == n,
                "mixed_attention: fp32 constants per head");
    return t->data_ptr<float>();
  };
  const float *p1 = vec(r1, Hs), *p2 = vec(r2, Hs), *ps = vec(sink, Ho), *pt = vec(talk, Ho * Hs);
  TORCH_CHECK((p1 == nullptr) == (p2 == nullptr), "mixed_attention: r1 and r2 go together");
  const int* cu = nullptr;
  if (cu_q.has_value()) {
    CHECK_I32(*cu_q);
    TORCH_CHECK(cu_q->numel() >= num_seqs + 1, "mixed_attention: cu_q [B + 1]");
    cu = cu_q->data_ptr<int>();
  } else {
    TORCH_CHECK(T == num_seqs * q_len, "mixed_attention: rows");
  }
  const int64_t pitch = (max_keys + 63) / 64 * 64;
  float* sp = nullptr;
  if (scratch.has_value()) {
    const int64_t need = cu ? tiles * 16 * Ho * pitch : T * splits * Ho * (v_cache.size(3) + 2);
    TORCH_CHECK(scratch->is_cuda() && scratch->is_contiguous() && (int64_t)scratch->nbytes() >= need * 4,
                "mixed_attention: scratch");
    sp = static_cast<float*>(scratch->data_ptr());
  }
  c10::cuda::CUDAGuard guard(q.device());
  check(b200_mixed_attention(q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(),
                             block_tables.data_ptr<int>(), cu, seq_lens.data_ptr<int>(), p1, p2, pt, ps, (int)num_seqs,
                             (int)T, (int)q_len, (int)max_keys, (int)block_tables.stride(0), (int)k_cache.size(2), (int)Hs,
                             (int)k_cache.size(1), (int)Ho, (int)v_cache.size(1), (int)head_dim, (int)head_dim_v,
                             (int)k_cache.size(3), (int)v_cache.size(3), q.stride(0), out.stride(0), (float)scale,
                             (float)softcap, (int)kind, (int)talk_terms, (int)splits, sp, (int)tile0, (int)tiles, pitch, f32 ? 1 : 0,
                             cur_stream()),
        "mixed_attention");
}

Tensor post_norm_residual(Tensor residual, const c10::optional<Tensor>& y, const c10::optional<Tensor>& w, int64_t groups,
                          double eps, int64_t true_width, const c10::optional<Tensor>& ids,
                          const c10::optional<Tensor>& table, const c10::optional<Tensor>& out_w, int64_t out_groups) {
  CHECK_ROWS(residual, at::kFloat);
  const int64_t T = residual.size(0), W = residual.size(1);
  const bool start = ids.has_value();
  TORCH_CHECK(start ? table.has_value() : y.has_value() && w.has_value(), "post_norm_residual: ids and table, or y and w");
  const Tensor& like = start ? *table : *y;
  const auto dt = like.scalar_type();
  const bool f32 = is_f32(like);
  CHECK_ROWS(like, dt);
  TORCH_CHECK(like.size(1) == W && (reinterpret_cast<uintptr_t>(like.data_ptr()) & 15) == 0, "post_norm_residual: rows [W]");
  const int* idp = nullptr;
  const void *wp = nullptr, *owp = nullptr;
  if (start) {
    CHECK_I32(*ids);
    TORCH_CHECK(ids->numel() >= T && like.is_contiguous(), "post_norm_residual: ids [T], table [rows, W]");
    idp = ids->data_ptr<int>();
  } else {
    TORCH_CHECK(like.size(0) == T, "post_norm_residual: y [T, W]");
    CHECK_VEC(*w, dt, W);
    wp = w->data_ptr();
  }
  if (out_w.has_value()) {
    CHECK_VEC(*out_w, dt, W);
    owp = out_w->data_ptr();
  }
  c10::cuda::CUDAGuard guard(residual.device());
  Tensor out = torch::empty({T, W}, like.options());
  check(b200_post_norm_residual(residual.data_ptr<float>(), residual.stride(0), idp, start ? like.data_ptr() : nullptr,
                                start ? (int)like.size(0) : 0, start ? nullptr : like.data_ptr(),
                                start ? 0 : like.stride(0), wp, (int)groups, owp, (int)out_groups, out.data_ptr(), W,
                                (float)eps, T, (int)W, (int)true_width, f32 ? 1 : 0, cur_stream()),
        "post_norm_residual");
  return out;
}

Tensor gelu_rows(const Tensor& z, const Tensor& ids, const Tensor& table, int64_t offset, int64_t dim) {
  const auto dt = z.scalar_type();
  const bool f32 = is_f32(z);
  CHECK_ROWS(z, dt);
  CHECK_ROWS(table, dt);
  CHECK_I32(ids);
  TORCH_CHECK(ids.numel() >= z.size(0) && z.size(1) >= dim && table.is_contiguous() && offset >= 0 &&
                  offset + dim <= table.size(1) && (reinterpret_cast<uintptr_t>(z.data_ptr()) & 15) == 0, "gelu_rows: shapes");
  c10::cuda::CUDAGuard guard(z.device());
  Tensor out = torch::empty({z.size(0), z.size(1)}, z.options());
  check(b200_gelu_rows(z.data_ptr(), z.stride(0), ids.data_ptr<int>(), table.data_ptr(), (int)table.size(0), table.stride(0),
                       (int)offset, (int)dim, (int)z.size(1), out.data_ptr(), (int)z.size(0), f32 ? 1 : 0, cur_stream()),
        "gelu_rows");
  return out;
}

void head_gemm(const Tensor& a, const Tensor& w, Tensor out) {
  const auto dt = a.scalar_type();
  const bool f32 = is_f32(a);
  TORCH_CHECK(a.is_cuda() && w.is_cuda() && out.is_cuda() && w.scalar_type() == dt && out.scalar_type() == dt &&
                  a.dim() == 3 && w.dim() == 3 && out.dim() == 3 && a.stride(2) == 1 && out.stride(2) == 1 &&
                  w.is_contiguous(), "head_gemm: a [T, H, K], w [H, N, K], out [T, H, N]");
  TORCH_CHECK(a.size(1) == w.size(0) && a.size(2) == w.size(2) && out.size(0) == a.size(0) &&
                  out.size(1) == a.size(1) && out.size(2) == w.size(1), "head_gemm: shapes");
  c10::cuda::CUDAGuard guard(a.device());
  check(b200_head_gemm(a.data_ptr(), a.stride(0), a.stride(1), w.data_ptr(), out.data_ptr(), out.stride(0),
                       out.stride(1), (int)a.size(0), (int)a.size(1), (int)w.size(1), (int)w.size(2), f32 ? 1 : 0,
                       cur_stream()),
        "head_gemm");
}

Tensor latent_gather(const Tensor& cache, const Tensor& block_tables, const Tensor& seq_lens, const Tensor& start,
                     int64_t num_seqs, int64_t total, int64_t max_len) {
  TORCH_CHECK(cache.is_cuda() && cache.is_contiguous() && cache.dim() == 3, "latent_gather: cache [blocks, size, row]");
  TORCH_CHECK(block_tables.is_cuda() && block_tables.scalar_type() == at::kInt && block_tables.dim() == 2 &&
                  block_tables.stride(1) == 1 && block_tables.size(0) >= num_seqs, "latent_gather: block tables");
  CHECK_I32(seq_lens);
  CHECK_I32(start);
  TORCH_CHECK(seq_lens.numel() >= num_seqs && start.numel() >= num_seqs, "latent_gather: sequences");
  c10::cuda::CUDAGuard guard(cache.device());
  Tensor out = torch::empty({total, cache.size(2)}, cache.options());
  check(b200_latent_gather(cache.data_ptr(), out.data_ptr(), block_tables.data_ptr<int>(), seq_lens.data_ptr<int>(),
                           start.data_ptr<int>(), (int)num_seqs, (int)max_len, (int)block_tables.stride(0),
                           (int)cache.size(1), (int)(cache.size(2) * cache.element_size()), (int)total, cur_stream()),
        "latent_gather");
  return out;
}

int64_t latent_decode_scratch_bytes(int64_t T, int64_t N, int64_t rank, int64_t splits) {
  return (int64_t)b200_latent_decode_scratch_bytes((int)T, (int)N, (int)rank, (int)splits);
}

void latent_decode(const Tensor& q, const Tensor& cache, const Tensor& block_tables, const Tensor& seq_lens,
                   int64_t num_seqs, int64_t heads, int64_t rank, double scale, int64_t splits,
                   const c10::optional<Tensor>& scratch, const Tensor& status, Tensor out) {
  TORCH_CHECK(q.is_cuda() && q.scalar_type() == at::kBFloat16 && q.is_contiguous() && q.dim() == 3 &&
                  cache.is_cuda() && cache.scalar_type() == at::kBFloat16 && cache.is_contiguous() && cache.dim() == 3 &&
                  out.is_cuda() && out.scalar_type() == at::kBFloat16 && out.is_contiguous(), "latent_decode: bf16");
  TORCH_CHECK(q.size(0) >= num_seqs && q.size(1) == heads && q.size(2) == cache.size(2) &&
                  out.numel() >= num_seqs * heads * rank, "latent_decode: shapes");
  TORCH_CHECK(block_tables.is_cuda() && block_tables.scalar_type() == at::kInt && block_tables.dim() == 2 &&
                  block_tables.stride(1) == 1 && block_tables.size(0) >= num_seqs, "latent_decode: block tables");
  CHECK_I32(seq_lens);
  void* sc = nullptr;
  if (splits > 1) {
    TORCH_CHECK(scratch.has_value() && (int64_t)scratch->nbytes() >=
                    latent_decode_scratch_bytes(num_seqs, heads, rank, splits), "latent_decode: scratch too small");
    sc = scratch->data_ptr();
  }
  c10::cuda::CUDAGuard guard(q.device());
  check(b200_latent_decode(q.data_ptr(), cache.data_ptr(), out.data_ptr(), block_tables.data_ptr<int>(),
                           seq_lens.data_ptr<int>(), (int)num_seqs, (int)heads, (int)cache.size(2), (int)rank,
                           (int)block_tables.stride(0), (int)cache.size(1), (int)cache.size(0), (float)scale,
                           (int)splits, sc, status.data_ptr<int>(), cur_stream()),
        "latent_decode");
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
  m.def("hyper_norm", &hyper_norm);
  m.def("gated_linear_prep", &gated_linear_prep);
  m.def("delta_prep", &delta_prep);
  m.def("recurrent_scan", &recurrent_scan);
  m.def("head_norm_gate", &head_norm_gate);
  m.def("token_mix", &token_mix);
  m.def("decay_prep", &decay_prep);
  m.def("qk_norm_rope", &qk_norm_rope);
  m.def("latent_prep", &latent_prep);
  m.def("mixed_attention_kind", &mixed_attention_kind);
  m.def("mixed_attention", &mixed_attention);
  m.def("post_norm_residual", &post_norm_residual);
  m.def("gelu_rows", &gelu_rows);
  m.def("head_gemm", &head_gemm);
  m.def("latent_gather", &latent_gather);
  m.def("latent_decode_scratch_bytes", &latent_decode_scratch_bytes);
  m.def("latent_decode", &latent_decode);
}

// Python bindings of the sm_100a extension.  With TK_SERVING_ONLY the module holds just what generation with a
// listed-layer stack launches (see ops/build.py): a box that only serves does not compile the training kernels, nor those of
// mechanisms that the model it serves does not have (TK_WITH_…).
#include <torch/extension.h>

#include "host.h"

namespace tk {
torch::Tensor gemm(const torch::Tensor&, const torch::Tensor&, const std::string&, const c10::optional<torch::Tensor>&, bool,
                   c10::optional<torch::ScalarType>);
std::vector<torch::Tensor> flash_attn_fwd(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, int64_t,
                                          bool, double, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&,
                                          const c10::optional<torch::Tensor>&, int64_t, int64_t, const c10::optional<torch::Tensor>&, double, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
torch::Tensor attention_packed(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, int64_t, double,
                               const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, int64_t, int64_t, double, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
torch::Tensor paged_attn_decode(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, double, int64_t, int64_t,
                                const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, double, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
std::vector<torch::Tensor> sample_tokens(const torch::Tensor&, double, int64_t, double, const torch::Tensor&);
std::vector<torch::Tensor> conv_heads(const torch::Tensor&, const c10::optional<torch::Tensor>&, const torch::Tensor&, int64_t, int64_t, int64_t, int64_t,
                                      double, double, int64_t, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, bool,
                                      const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&,
                                      const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, bool);
torch::Tensor stream_rmsnorm(torch::Tensor, const torch::Tensor&, double, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&,
                             const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, double, double);
torch::Tensor stream_joined_rmsnorm(torch::Tensor, const torch::Tensor&, double, double, const torch::Tensor&, const c10::optional<torch::Tensor>&,
                                    const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
torch::Tensor rotary_table(const torch::Tensor&, const torch::Tensor&);
std::vector<torch::Tensor> rotary_heads(const torch::Tensor&, int64_t, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&,
                                        const torch::Tensor&, int64_t, int64_t, bool, int64_t, int64_t, int64_t, int64_t, double, const c10::optional<torch::Tensor>&,
                                        const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, bool);
torch::Tensor latent_rotary(const torch::Tensor&, int64_t, int64_t, int64_t, int64_t, int64_t, int64_t, const c10::optional<torch::Tensor>&, double,
                            const c10::optional<torch::Tensor>&, int64_t, int64_t, bool, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&,
                            const c10::optional<torch::Tensor>&, bool);
torch::Tensor stream_gated_rmsnorm(torch::Tensor, const torch::Tensor&, double, double, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&,
                                   const torch::Tensor&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
std::vector<torch::Tensor> latent_norms(const torch::Tensor&, int64_t, int64_t, const torch::Tensor&, int64_t, int64_t, const c10::optional<torch::Tensor>&, double,
                                        const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
torch::Tensor latent_decode(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, double, const c10::optional<torch::Tensor>&,
                            const c10::optional<torch::Tensor>&, int64_t, int64_t);
torch::Tensor hgrn2_prefill(const torch::Tensor&, int64_t, int64_t, int64_t, int64_t, int64_t, int64_t, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&,
                            double, const torch::Tensor&, int64_t, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
torch::Tensor hgrn2_step(const torch::Tensor&, int64_t, int64_t, int64_t, int64_t, int64_t, int64_t, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&,
                         double, const torch::Tensor&, const torch::Tensor&);
std::vector<torch::Tensor> moe_topk(const torch::Tensor&, const c10::optional<torch::Tensor>&, int64_t, const c10::optional<torch::Tensor>&, int64_t, int64_t, double,
                                    const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
std::vector<torch::Tensor> moe_group_rows(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&);
torch::Tensor grouped_gemm_f32(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, bool);
torch::Tensor head_gemm(const torch::Tensor&, const torch::Tensor&, bool, const c10::optional<torch::Tensor>&);
torch::Tensor grouped_gemm(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const std::string&, const c10::optional<torch::Tensor>&,
                           const c10::optional<torch::Tensor>&, bool, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&,
                           const c10::optional<std::string>&);
torch::Tensor glu_columns(const torch::Tensor&, int64_t, int64_t, int64_t, double, bool);
torch::Tensor stream_normed(torch::Tensor, const c10::optional<torch::Tensor>&, double, const torch::Tensor&, const c10::optional<torch::Tensor>&, const torch::Tensor&, const c10::optional<torch::Tensor>&,
                            const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
torch::Tensor embed_positions(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&);
std::vector<torch::Tensor> plain_heads(const torch::Tensor&, int64_t, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, bool, bool, int64_t,
                                       int64_t, int64_t, int64_t, double, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&, bool);
torch::Tensor conv_silu(const torch::Tensor&, int64_t, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, bool, const c10::optional<torch::Tensor>&,
                        const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
torch::Tensor selective_prefill(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, int64_t, int64_t, const torch::Tensor&,
                                const torch::Tensor&, int64_t, const torch::Tensor&, int64_t, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
torch::Tensor selective_step(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, int64_t, int64_t, const torch::Tensor&,
                             const torch::Tensor&, int64_t, const torch::Tensor&, const torch::Tensor&);
torch::Tensor mlstm_prefill(const torch::Tensor&, int64_t, int64_t, int64_t, int64_t, const torch::Tensor&, const torch::Tensor&, double, const torch::Tensor&, double,
                            const torch::Tensor&, int64_t, const c10::optional<torch::Tensor>&, const c10::optional<torch::Tensor>&);
torch::Tensor mlstm_step(const torch::Tensor&, int64_t, int64_t, int64_t, int64_t, const torch::Tensor&, const torch::Tensor&, double, const torch::Tensor&, double,
                         const torch::Tensor&, const torch::Tensor&);
void set_gemm_pair(int64_t);
void set_gemm_staged(int64_t);
#ifndef TK_SERVING_ONLY
torch::Tensor grouped_gemm_wgrad(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, int64_t);
std::vector<torch::Tensor> rmsnorm_fwd(const torch::Tensor&, const torch::Tensor&, double, double, const c10::optional<torch::Tensor>&);
std::vector<torch::Tensor> rmsnorm_bwd(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, double,
                                       const c10::optional<torch::Tensor>&);
std::vector<torch::Tensor> qk_norm_rope_fwd(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&,
                                            const torch::Tensor&, int64_t, int64_t, int64_t, double);
std::vector<torch::Tensor> qk_norm_rope_bwd(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&,
                                            const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&,
                                            const torch::Tensor&, int64_t, int64_t, int64_t);
torch::Tensor swiglu_fwd(const torch::Tensor&);
torch::Tensor swiglu_bwd(const torch::Tensor&, const torch::Tensor&);
torch::Tensor geglu_fwd(const torch::Tensor&);
torch::Tensor geglu_bwd(const torch::Tensor&, const torch::Tensor&);
void adamw_step(torch::Tensor, torch::Tensor, torch::Tensor, const torch::Tensor&, const c10::optional<torch::Tensor>&, double, double,
                double, double, double, int64_t, double);
torch::Tensor sumsq(const torch::Tensor&);
std::vector<torch::Tensor> logprob_fwd(const torch::Tensor&, const torch::Tensor&, double, bool);
torch::Tensor logprob_bwd(torch::Tensor, const torch::Tensor&, const torch::Tensor&, const c10::optional<torch::Tensor>&,
                          const torch::Tensor&, const c10::optional<torch::Tensor>&, double);
std::vector<torch::Tensor> flash_attn_bwd(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&,
                                          const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, int64_t, bool, double,
                                          const c10::optional<torch::Tensor>&, int64_t);
std::tuple<torch::Tensor, py::bytes, int64_t> symm_alloc(int64_t);
int64_t symm_open(const py::bytes&);
void symm_close(int64_t);
void symm_barrier(const std::vector<int64_t>&, int64_t, int64_t, int64_t);
void peer_all_gather(torch::Tensor, const std::vector<int64_t>&, int64_t, int64_t, int64_t);
void peer_pull(const std::vector<int64_t>&, const std::vector<int64_t>&, const std::vector<int64_t>&, const std::vector<int64_t>&,
               const std::vector<int64_t>&, const std::vector<int64_t>&, int64_t);
void peer_reduce_scatter_acc(torch::Tensor, const std::vector<int64_t>&, int64_t, double, const c10::optional<torch::Tensor>&, int64_t);
void ulysses_exchange(const torch::Tensor&, const std::vector<int64_t>&, int64_t, bool, int64_t);
void peer_copy_cast(const torch::Tensor&, const std::vector<int64_t>&, int64_t);
torch::Tensor causal_conv1d_fwd(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, bool);
std::vector<torch::Tensor> gdn_recurrent_fwd(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&, const torch::Tensor&,
                                             const torch::Tensor&, const torch::Tensor&, const c10::optional<torch::Tensor>&, double, bool);
std::vector<torch::Tensor> moe_router(const torch::Tensor&, int64_t, bool);
void gemm_rs(const torch::Tensor&, const torch::Tensor&, const std::string&, const std::vector<int64_t>&, int64_t);
void gemm_head_scatter(const torch::Tensor&, const torch::Tensor&, const std::vector<int64_t>&, int64_t, int64_t, int64_t, int64_t);
std::vector<torch::Tensor> gemm_ag(const std::vector<int64_t>&, int64_t, const torch::Tensor&, const std::string&, int64_t, const torch::Tensor&, int64_t, int64_t);
torch::Tensor tp_stage_reduce(const torch::Tensor&);
torch::Tensor moe_rows_gather(const torch::Tensor&, const torch::Tensor&, const c10::optional<torch::Tensor>&);
torch::Tensor moe_rows_combine(const torch::Tensor&, const torch::Tensor&, const c10::optional<torch::Tensor>&);
torch::Tensor moe_combine_wgrad(const torch::Tensor&, const torch::Tensor&, const torch::Tensor&);
torch::Tensor ep_rows_gather(const std::vector<int64_t>&, const std::vector<int64_t>&, const std::vector<int64_t>&, const torch::Tensor&, const torch::Tensor&, int64_t,
                             const torch::Tensor&, int64_t, int64_t);
torch::Tensor ep_rows_combine(const std::vector<int64_t>&, const torch::Tensor&, const torch::Tensor&, const c10::optional<torch::Tensor>&, int64_t, int64_t);
torch::Tensor ep_combine_wgrad(const torch::Tensor&, const std::vector<int64_t>&, const torch::Tensor&, const torch::Tensor&, int64_t);
#endif
}  // namespace tk

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.def("gemm", &tk::gemm, py::arg("a"), py::arg("b"), py::arg("layout") = "nt", py::arg("out") = py::none(),
        py::arg("accumulate") = false, py::arg("out_dtype") = py::none());
  m.def("flash_attn_fwd", &tk::flash_attn_fwd, py::arg("q"), py::arg("k"), py::arg("v"), py::arg("cu"), py::arg("max_seqlen"), py::arg("causal"),
        py::arg("scale"), py::arg("cu_k") = py::none(), py::arg("sinks") = py::none(), py::arg("gate") = py::none(), py::arg("window") = 0, py::arg("chunk") = 0,
        py::arg("key_tail") = py::none(), py::arg("cap") = 0.0, py::arg("temp") = py::none(), py::arg("slope") = py::none(),
        py::arg("rate") = py::none(), py::arg("table") = py::none(), py::arg("bucket") = py::none());
  m.def("paged_attn_decode", &tk::paged_attn_decode, py::arg("q"), py::arg("k"), py::arg("v"), py::arg("tables"), py::arg("seq_lens"), py::arg("scale"),
        py::arg("window") = 0, py::arg("chunk") = 0, py::arg("sinks") = py::none(), py::arg("gate") = py::none(), py::arg("cap") = 0.0, py::arg("temp") = py::none(), py::arg("slope") = py::none(),
        py::arg("rate") = py::none(), py::arg("table") = py::none(), py::arg("bucket") = py::none());
  m.def("sample_tokens", &tk::sample_tokens);
  m.def("set_gemm_pair", &tk::set_gemm_pair);
  m.def("set_gemm_staged", &tk::set_gemm_staged);
  m.def("read_and_clear_error", &tk::read_and_clear_error, "Value of the device error word (0 = healthy); clears it.");
  m.def("num_sms", &tk::num_sms);
  m.def("launch_count", &tk::launch_count, "Number of kernels launched by this extension so far.");
  m.def("attention_packed", &tk::attention_packed, py::arg("q"), py::arg("k"), py::arg("v"), py::arg("cu"), py::arg("max_seqlen"), py::arg("scale"),
        py::arg("sinks") = py::none(), py::arg("gate") = py::none(), py::arg("window") = 0, py::arg("chunk") = 0, py::arg("cap") = 0.0, py::arg("temp") = py::none(), py::arg("slope") = py::none(),
        py::arg("rate") = py::none(), py::arg("table") = py::none(), py::arg("bucket") = py::none());
#ifdef TK_WITH_CONVOLUTION
  m.def("conv_heads", &tk::conv_heads, py::arg("proj"), py::arg("weight"), py::arg("pos"), py::arg("hq"), py::arg("hkv"), py::arg("d"), py::arg("e"), py::arg("eps"),
        py::arg("coef") = 0.0, py::arg("every") = 0, py::arg("v_first") = py::none(), py::arg("lam") = py::none(), py::arg("step") = false,
        py::arg("hist") = py::none(), py::arg("slot") = py::none(), py::arg("left") = py::none(), py::arg("pool_row") = py::none(),
        py::arg("k_pool") = py::none(), py::arg("v_pool") = py::none(), py::arg("want_k") = true);
#endif
#ifdef TK_WITH_HEADS
  m.def("plain_heads", &tk::plain_heads);
#endif
#ifdef TK_WITH_SELECTIVE
  m.def("conv_silu", &tk::conv_silu);
  m.def("selective_prefill", &tk::selective_prefill);
  m.def("selective_step", &tk::selective_step);
#endif
#ifdef TK_WITH_MEMORY
  m.def("mlstm_prefill", &tk::mlstm_prefill);
  m.def("mlstm_step", &tk::mlstm_step);
#endif
#ifdef TK_WITH_ROTARY
  m.def("rotary_table", &tk::rotary_table);
  m.def("rotary_heads", &tk::rotary_heads);
  m.def("latent_rotary", &tk::latent_rotary);
#endif
  m.def("stream_rmsnorm", &tk::stream_rmsnorm, py::arg("x"), py::arg("w"), py::arg("eps"), py::arg("y1") = py::none(), py::arg("s1") = py::none(),
        py::arg("y2") = py::none(), py::arg("s2") = py::none(), py::arg("mult") = 1.0, py::arg("offset") = 0.0);
  m.def("stream_gated_rmsnorm", &tk::stream_gated_rmsnorm);
  m.def("stream_normed", &tk::stream_normed);
  m.def("embed_positions", &tk::embed_positions);
  m.def("stream_joined_rmsnorm", &tk::stream_joined_rmsnorm, py::arg("x"), py::arg("w"), py::arg("eps"), py::arg("offset"), py::arg("y"), py::arg("row_of") = py::none(),
        py::arg("share") = py::none(), py::arg("beside") = py::none(), py::arg("open") = py::none());
#ifdef TK_WITH_LATENT
  m.def("latent_norms", &tk::latent_norms);
  m.def("latent_decode", &tk::latent_decode, py::arg("q"), py::arg("pool"), py::arg("tables"), py::arg("lens"), py::arg("scale"), py::arg("sinks"), py::arg("gate"),
        py::arg("rank"), py::arg("window") = 0);
#endif
#ifdef TK_WITH_RECURRENT
  m.def("hgrn2_prefill", &tk::hgrn2_prefill);
  m.def("hgrn2_step", &tk::hgrn2_step);
#endif
#ifdef TK_WITH_EXPERTS
  m.def("moe_topk", &tk::moe_topk, py::arg("logits"), py::arg("bias"), py::arg("k"), py::arg("forced") = py::none(), py::arg("groups") = 0, py::arg("keep") = 0,
        py::arg("factor") = 1.0, py::arg("x") = py::none(), py::arg("shared") = py::none());
  m.def("moe_group_rows", &tk::moe_group_rows);
  m.def("grouped_gemm_f32", &tk::grouped_gemm_f32);
#endif
  m.def("head_gemm", &tk::head_gemm, py::arg("x"), py::arg("w"), py::arg("nn"), py::arg("out") = py::none());
  m.def("grouped_gemm", &tk::grouped_gemm, py::arg("x"), py::arg("w"), py::arg("offsets"), py::arg("layout") = "nt", py::arg("group_map") = py::none(),
        py::arg("out") = py::none(), py::arg("accumulate") = false, py::arg("x2") = py::none(), py::arg("w2") = py::none(), py::arg("act") = py::none());
  m.def("glu_columns", &tk::glu_columns, py::arg("p"), py::arg("gate"), py::arg("up"), py::arg("width"), py::arg("limit") = 0.0, py::arg("gelu") = false);
#ifndef TK_SERVING_ONLY
  m.def("grouped_gemm_wgrad", &tk::grouped_gemm_wgrad);
  m.def("rmsnorm_fwd", &tk::rmsnorm_fwd, py::arg("x"), py::arg("w"), py::arg("eps"), py::arg("offset"), py::arg("residual") = py::none());
  m.def("rmsnorm_bwd", &tk::rmsnorm_bwd, py::arg("g"), py::arg("x"), py::arg("w"), py::arg("rstd"), py::arg("offset"),
        py::arg("gadd") = py::none());
  m.def("qk_norm_rope_fwd", &tk::qk_norm_rope_fwd);
  m.def("qk_norm_rope_bwd", &tk::qk_norm_rope_bwd);
  m.def("swiglu_fwd", &tk::swiglu_fwd);
  m.def("swiglu_bwd", &tk::swiglu_bwd);
  m.def("geglu_fwd", &tk::geglu_fwd);
  m.def("geglu_bwd", &tk::geglu_bwd);
  m.def("adamw_step", &tk::adamw_step);
  m.def("sumsq", &tk::sumsq);
  m.def("logprob_fwd", &tk::logprob_fwd);
  m.def("logprob_bwd", &tk::logprob_bwd);
  m.def("flash_attn_bwd", &tk::flash_attn_bwd, py::arg("dout"), py::arg("q"), py::arg("k"), py::arg("v"), py::arg("out"), py::arg("lse"), py::arg("cu"),
        py::arg("max_seqlen"), py::arg("causal"), py::arg("scale"), py::arg("cu_k") = py::none(), py::arg("max_seqlen_k") = 0);
  m.def("symm_alloc", &tk::symm_alloc, "cudaMalloc'ed uint8 tensor + its CUDA IPC handle");
  m.def("symm_open", &tk::symm_open);
  m.def("symm_close", &tk::symm_close);
  m.def("symm_barrier", &tk::symm_barrier, py::arg("flag_ptrs"), py::arg("rank"), py::arg("epoch"), py::arg("timeout_ms") = 3000);
  m.def("peer_all_gather", &tk::peer_all_gather);
  m.def("peer_pull", &tk::peer_pull, py::arg("src"), py::arg("dst"), py::arg("src_stride"), py::arg("dst_stride"), py::arg("chunk_bytes"),
        py::arg("rows"), py::arg("blocks_per_job"));
  m.def("peer_reduce_scatter_acc", &tk::peer_reduce_scatter_acc);
  m.def("ulysses_exchange", &tk::ulysses_exchange);
  m.def("peer_copy_cast", &tk::peer_copy_cast);
  m.def("causal_conv1d_fwd", &tk::causal_conv1d_fwd);
  m.def("gdn_recurrent_fwd", &tk::gdn_recurrent_fwd, py::arg("q"), py::arg("k"), py::arg("v"), py::arg("g"), py::arg("beta"), py::arg("cu"),
        py::arg("init_state") = py::none(), py::arg("scale") = 1.0, py::arg("want_state") = false);
  m.def("moe_router", &tk::moe_router);
  m.def("gemm_rs", &tk::gemm_rs);
  m.def("gemm_head_scatter", &tk::gemm_head_scatter);
  m.def("gemm_ag", &tk::gemm_ag);
  m.def("tp_stage_reduce", &tk::tp_stage_reduce);
  m.def("moe_rows_gather", &tk::moe_rows_gather);
  m.def("moe_rows_combine", &tk::moe_rows_combine);
  m.def("moe_combine_wgrad", &tk::moe_combine_wgrad);
  m.def("ep_rows_gather", &tk::ep_rows_gather);
  m.def("ep_rows_combine", &tk::ep_rows_combine);
  m.def("ep_combine_wgrad", &tk::ep_combine_wgrad);
#endif
}

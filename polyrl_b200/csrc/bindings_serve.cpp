// polyrl_b200 — bindings of the serving core (module ``_serve``): native scheduler and page manager, dense GEMMs, packed
// attention, sampling and the sequence-mixer kernels.  Everything a rollout engine of a mixer stack needs is in this one
// module, so a serving host builds it without the training and multi-GPU kernels of ``_C``.
#include "bindings_common.hpp"
#include "kv_manager.hpp"
#include "scheduler.hpp"

extern "C" {
int prl_gemm_bf16(const void*, const void*, void*, const void*, int, int, int, int64_t, int64_t, int64_t, int, cudaStream_t);
int prl_sample(const void*, int, int64_t, int, int, const float*, const uint64_t*, int, int64_t*, float*, cudaStream_t);
int prl_sample_topk_topp(const void*, int, int64_t, int, int, const float*, const uint64_t*, int, int, float, int64_t*, float*, cudaStream_t);
int prl_attn_fwd(const void*, const void*, const void*, void*, float*, const int32_t*, const int32_t*, int, int, int, int, int, int, int, int64_t, int64_t, int64_t, int64_t, float, int, int, const float*, int, int, long long*, cudaStream_t);
int prl_paged_decode_workspace_floats(int, int, int, int);
int prl_paged_decode(const void*, int64_t, const void*, const void*, const int32_t*, int64_t, const int32_t*, int, int, int, int, float, int, int, int, float*, void*, int64_t, cudaStream_t);
int prl_gemm_clamped_glu_bf16(const void*, const void*, void*, int, int, int, int64_t, int64_t, int64_t, float, float, cudaStream_t);
int prl_gemm_swiglu_bf16(const void*, const void*, void*, void*, int, int, int, int64_t, int64_t, int64_t, int64_t, cudaStream_t);
int prl_gemm_experts_bf16(const void*, const void*, void*, const int32_t*, int, int, int, int, int, float, float, cudaStream_t);
int prl_sink_decode(const void*, const void*, const void*, const int32_t*, int64_t, const int32_t*, int, int, int, int, int, float, int, const float*, float*, void*, cudaStream_t);
int prl_map_attn_fwd(const void*, const void*, const void*, void*, const int32_t*, const int32_t*, int, int, int, int, int, int, int, int, int, float, int, const float*, float, float, int, cudaStream_t);
int prl_map_decode_ok(int, int, int);
int prl_map_decode(const void*, const void*, const void*, const int32_t*, int64_t, const int32_t*, int, int, int, int, int, int, float, int, int, const float*, float, float, float*, void*, cudaStream_t);
int prl_gemm_gelu_bf16(const void*, const void*, void*, int, int, int, int64_t, int64_t, int64_t, int, cudaStream_t);
int prl_mix_embed(const int64_t*, const void*, const float*, float*, void*, int, int, float, int, cudaStream_t);
int prl_mix_norm_add(const void*, int64_t, float*, const float*, const float*, void*, int, int, float, int, cudaStream_t);
int prl_mix_rms(const float*, const float*, void*, int, int, float, int, int, cudaStream_t);
int prl_mix_gated_norm(const void*, int64_t, const void*, int64_t, const float*, void*, int64_t, int, int, int, float, int, int, cudaStream_t);
int prl_mix_conv(const void*, int64_t, const float*, const float*, void*, const int32_t*, const int32_t*, const int64_t*, const int32_t*, void*, int64_t, int, int, int, int, int, cudaStream_t);
int prl_mix_latent_prep(const void*, int64_t, int, int, int, const float*, const float*, const double*, const int64_t*, const int64_t*, void*, void*, void*, int, float, int, cudaStream_t);
int prl_mix_rope(void*, int64_t, int, int, int, int, const double*, const int64_t*, int, int, cudaStream_t);
int prl_mix_gelu(void*, int64_t, int, int, cudaStream_t);
int prl_mix_turn_rows(const void*, int64_t, const float*, const double*, const double*, const int64_t*, const int64_t*, void*, void*, void*, void*, void*, int, int, int, int, int, int, int, int, float, int, cudaStream_t);
int prl_mix_turn_back(const void*, const void*, int64_t, const double*, const int64_t*, float, void*, int64_t, int, int, int, int, int, cudaStream_t);
int prl_mix_qk_prep(const void*, int64_t, int, int, int, int, int, const float*, const float*, const double*, const int64_t*, const int64_t*, void*, void*, void*, void*, void*, int, float, int, cudaStream_t);
int prl_mix_gather_keys(const void*, const void*, const int64_t*, void*, void*, int64_t, int, int, int, cudaStream_t);
int prl_mix_map_rows(const void*, int64_t, const float*, const float*, const float*, const double*, const int64_t*, const int64_t*, void*, void*, void*, void*, void*, int, int, int, int, int, int, int, int, int, float, int, cudaStream_t);
int prl_mix_input_conv(const void*, int64_t, const float*, const float*, void*, const int32_t*, const int32_t*, const int64_t*, const int32_t*, void*, void*, int, int, int, int, int, cudaStream_t);
int prl_mix_poly_norm(const void*, int64_t, const float*, void*, int, int, float, int, cudaStream_t);
int prl_mix_silu_glu(const void*, void*, int64_t, int, int, int, cudaStream_t);
int prl_mix_route_tiles(int64_t, int64_t);
int prl_mix_route(const float*, int64_t, int, int, int, int32_t*, float*, int32_t*, int32_t*, int32_t*, int, cudaStream_t);
int prl_mix_expert_rows(const void*, int64_t, const int32_t*, const float*, const int32_t*, const int32_t*, void*, int32_t*, int, int, int, int, cudaStream_t);
int prl_mix_expert_gemm(const void*, const void*, const int32_t*, void*, int, int, int, int, int, cudaStream_t);
int prl_mix_clamped_glu(const void*, void*, int64_t, int, int, float, float, int, cudaStream_t);
int prl_mix_delta_ok(const void*, int64_t, const void*, int64_t, const void*, int64_t, int, int);
int64_t prl_mix_delta_chunks(int64_t, int64_t);
int prl_mix_delta_work_bytes();
int prl_mix_delta_gate_floats();
int prl_mix_chunk_supported(int);
int prl_mix_latent_tc_ok(int, int);
}
#include "mix_params.hpp"
extern "C" {
int prl_mix_scan(const prl::ScanParams*, int, int, int, cudaStream_t);
int prl_mix_chunk(const prl::ScanParams*, int, cudaStream_t);
int prl_mix_chunk_tc_ok(const prl::ScanParams*);
int prl_mix_chunk_tc(const prl::ScanParams*, int, int32_t*, cudaStream_t);
int prl_mix_latent(const prl::LatentParams*, int, int, cudaStream_t);
int prl_mix_window(const prl::WindowParams*, int, cudaStream_t);
int prl_mix_block(const prl::BlockParams*, int, cudaStream_t);
int prl_mix_gla_ok(const prl::ScanParams*);
int64_t prl_mix_gla_chunks(int64_t, int64_t);
int64_t prl_mix_gla_work_bytes(int);
int64_t prl_mix_gla_keep_floats(int);
int prl_mix_gla(const prl::ScanParams*, int64_t, int64_t, void*, float*, int32_t*, cudaStream_t);
int prl_mix_sink(const prl::SinkParams*, int, cudaStream_t);
int prl_mix_selective(const prl::SelectiveParams*, int, int, cudaStream_t);
int prl_mix_streams(const prl::StreamsParams*, int, cudaStream_t);
int prl_mix_map_attention(const prl::MapParams*, int, cudaStream_t);
int prl_mix_delta(const prl::ScanParams*, int64_t, int64_t, void*, float*, int32_t*, cudaStream_t);
}

namespace {

at::Tensor gemm_bf16(const at::Tensor& a, const at::Tensor& b, const c10::optional<at::Tensor>& residual,
                     c10::optional<at::Tensor> out, int64_t force_bn) {
  CHECK_BF16(a); CHECK_BF16(b);
  TORCH_CHECK(a.dim() == 2 && b.dim() == 2 && a.size(1) == b.size(1), "gemm_bf16: A[M,K] B[N,K]");
  CHECK_LASTDIM(a); CHECK_LASTDIM(b);
  const int M = a.size(0), K = a.size(1), N = b.size(0);
  TORCH_CHECK(K % 8 == 0 && N % 8 == 0, "K and N must be multiples of 8");
  TORCH_CHECK(a.stride(0) % 8 == 0 && b.stride(0) % 8 == 0, "row pitch must be a multiple of 8 elements");
  c10::cuda::CUDAGuard g(a.device());
  at::Tensor d = out.has_value() ? *out : at::empty({M, N}, a.options());
  CHECK_BF16(d); CHECK_LASTDIM(d);
  const void* r = nullptr;
  if (residual.has_value()) {
    CHECK_BF16(*residual);
    TORCH_CHECK(residual->sizes() == d.sizes() && residual->stride(0) == d.stride(0) && residual->stride(1) == 1);
    r = residual->data_ptr();
  }
  check(prl_gemm_bf16(a.data_ptr(), b.data_ptr(), d.data_ptr(), r, M, N, K, a.stride(0), b.stride(0), d.stride(0),
                      static_cast<int>(force_bn), cur_stream()), "gemm_bf16");
  return d;
}

std::vector<at::Tensor> sample(const at::Tensor& logits, const c10::optional<at::Tensor>& inv_temp,
                               const c10::optional<at::Tensor>& seeds, bool greedy) {
  TORCH_CHECK(logits.is_cuda() && logits.dim() == 2 && logits.stride(1) == 1);
  const int dt = logits.scalar_type() == at::kFloat ? 0 : 1;
  TORCH_CHECK(dt == 0 || logits.scalar_type() == at::kBFloat16);
  const int B = logits.size(0), V = logits.size(1);
  c10::cuda::CUDAGuard g(logits.device());
  at::Tensor tok = at::empty({B}, logits.options().dtype(at::kLong));
  at::Tensor lp = at::empty({B}, logits.options().dtype(at::kFloat));
  const uint64_t* sd = nullptr;
  if (seeds.has_value()) { TORCH_CHECK(seeds->scalar_type() == at::kLong); sd = reinterpret_cast<const uint64_t*>(seeds->data_ptr<int64_t>()); }
  check(prl_sample(logits.data_ptr(), dt, logits.stride(0), B, V,
                   inv_temp.has_value() ? inv_temp->data_ptr<float>() : nullptr, sd, greedy ? 1 : 0,
                   tok.data_ptr<int64_t>(), lp.data_ptr<float>(), cur_stream()), "sample");
  return {tok, lp};
}

std::vector<at::Tensor> sample_topk_topp(const at::Tensor& logits, const c10::optional<at::Tensor>& inv_temp,
                                         const c10::optional<at::Tensor>& seeds, bool greedy, int64_t top_k, double top_p) {
  TORCH_CHECK(logits.is_cuda() && logits.dim() == 2 && logits.stride(1) == 1);
  const int dt = logits.scalar_type() == at::kFloat ? 0 : 1;
  TORCH_CHECK(dt == 0 || logits.scalar_type() == at::kBFloat16);
  const int B = logits.size(0), V = logits.size(1);
  c10::cuda::CUDAGuard g(logits.device());
  at::Tensor tok = at::empty({B}, logits.options().dtype(at::kLong));
  at::Tensor lp = at::empty({B}, logits.options().dtype(at::kFloat));
  const uint64_t* sd = nullptr;
  if (seeds.has_value()) { TORCH_CHECK(seeds->scalar_type() == at::kLong); sd = reinterpret_cast<const uint64_t*>(seeds->data_ptr<int64_t>()); }
  check(prl_sample_topk_topp(logits.data_ptr(), dt, logits.stride(0), B, V,
                             inv_temp.has_value() ? inv_temp->data_ptr<float>() : nullptr, sd, greedy ? 1 : 0,
                             static_cast<int>(top_k), static_cast<float>(top_p), tok.data_ptr<int64_t>(), lp.data_ptr<float>(),
                             cur_stream()), "sample_topk_topp");
  return {tok, lp};
}

std::vector<at::Tensor> attn_fwd(const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, const at::Tensor& cu_q,
                                 const at::Tensor& cu_k, double sm_scale, bool causal, bool want_lse,
                                 const c10::optional<at::Tensor>& dbg, const c10::optional<at::Tensor>& sink, int64_t window, int64_t keep_first) {
  CHECK_BF16(q); CHECK_BF16(k); CHECK_BF16(v);
  const int64_t dk = q.size(-1), dv = v.size(-1);
  TORCH_CHECK(q.dim() == 3 && k.dim() == 3 && v.dim() == 3 && (dk == 64 || dk == 128 || dk == 192) && k.size(2) == dk && (dv == 128 || (dv == 64 && dk != 192)) &&
              v.size(1) == k.size(1) && v.size(0) == k.size(0), "attn_fwd: query / key width 64, 128 or 192, value width 64 or 128");
  TORCH_CHECK(window >= 0 && window <= 0x7fffffff && keep_first >= 0 && keep_first <= 0x7fffff00 && (window == 0 || causal), "attn_fwd: window");
  TORCH_CHECK(q.stride(2) == 1 && q.stride(1) == dk && k.stride(2) == 1 && k.stride(1) == dk && v.stride(2) == 1 && v.stride(1) == dv,
              "attn_fwd: heads must be contiguous inside a token row");
  TORCH_CHECK(q.stride(0) % 8 == 0 && k.stride(0) % 8 == 0 && v.stride(0) % 8 == 0);
  TORCH_CHECK((reinterpret_cast<uintptr_t>(q.data_ptr()) & 15) == 0 && (reinterpret_cast<uintptr_t>(k.data_ptr()) & 15) == 0 &&
              (reinterpret_cast<uintptr_t>(v.data_ptr()) & 15) == 0, "attn_fwd: 16-byte aligned operands");
  TORCH_CHECK(cu_q.is_cuda() && cu_q.scalar_type() == at::kInt && cu_q.is_contiguous() && cu_k.is_cuda() &&
              cu_k.scalar_type() == at::kInt && cu_k.is_contiguous() && cu_q.numel() == cu_k.numel());
  const int Tq = q.size(0), Tk = k.size(0), nq = q.size(1), nkv = k.size(1), B = cu_q.numel() - 1;
  if (sink.has_value()) { CHECK_F32(*sink); TORCH_CHECK(sink->is_contiguous() && sink->numel() == nq); }
  c10::cuda::CUDAGuard g(q.device());
  at::Tensor o = at::empty({Tq, nq, dv}, q.options());
  at::Tensor lse = want_lse ? at::empty({nq, Tq}, q.options().dtype(at::kFloat)) : at::Tensor();
  check(prl_attn_fwd(q.data_ptr(), k.data_ptr(), v.data_ptr(), o.data_ptr(), want_lse ? lse.data_ptr<float>() : nullptr,
                     cu_q.data_ptr<int>(), cu_k.data_ptr<int>(), B, Tq, Tk, nq, nkv, static_cast<int>(dk), static_cast<int>(dv), q.stride(0), k.stride(0), v.stride(0),
                     static_cast<int64_t>(nq) * dv, static_cast<float>(sm_scale), causal ? 1 : 0, Tq / 128 + B,
                     sink.has_value() ? sink->data_ptr<float>() : nullptr, static_cast<int>(window), static_cast<int>(keep_first),
                     dbg.has_value() ? reinterpret_cast<long long*>(dbg->data_ptr<int64_t>()) : nullptr, cur_stream()),
        "attn_fwd");
  if (want_lse) return {o, lse};
  return {o};
}

at::Tensor paged_decode(const at::Tensor& q, const at::Tensor& k_cache, const at::Tensor& v_cache,
                        const at::Tensor& block_table, const at::Tensor& seq_lens, int64_t nq, int64_t nkv, int64_t d,
                        double sm_scale, int64_t splits, c10::optional<at::Tensor> out, int64_t window, int64_t keep_first) {
  CHECK_BF16(q); CHECK_BF16(k_cache); CHECK_BF16(v_cache);
  TORCH_CHECK(block_table.scalar_type() == at::kInt && seq_lens.scalar_type() == at::kInt);
  TORCH_CHECK(q.dim() == 2 && q.stride(1) == 1 && k_cache.is_contiguous() && v_cache.is_contiguous());
  TORCH_CHECK(k_cache.size(2) == 16, "KV page size must be 16 tokens");
  TORCH_CHECK(window >= 0 && window <= 0x7fffffff && keep_first >= 0 && keep_first <= 0x7fffff00, "paged_decode: window");
  const int B = q.size(0);
  c10::cuda::CUDAGuard g(q.device());
  at::Tensor o = out.has_value() ? *out : at::empty({B, nq * d}, q.options());
  const int64_t ws = prl_paged_decode_workspace_floats(B, nq, d, splits);
  at::Tensor workspace = at::empty({ws}, q.options().dtype(at::kFloat));
  check(prl_paged_decode(q.data_ptr(), q.stride(0), k_cache.data_ptr(), v_cache.data_ptr(),
                         block_table.data_ptr<int32_t>(), block_table.stride(0), seq_lens.data_ptr<int32_t>(), B, nq,
                         nkv, d, static_cast<float>(sm_scale), splits, static_cast<int>(window), static_cast<int>(keep_first),
                         workspace.data_ptr<float>(), o.data_ptr(), o.stride(0), cur_stream()), "paged_decode");
  return o;
}

static at::Tensor vec_i64(const std::vector<int64_t>& v) {
  return at::tensor(c10::ArrayRef<int64_t>(v.data(), v.size()), at::TensorOptions().dtype(at::kLong));
}

// ---------------------------------------------------------------------------------------------- sequence mixers
int dt_of(const at::Tensor& t, const char* what) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == at::kBFloat16 || t.scalar_type() == at::kFloat), what, ": CUDA bf16 or fp32 tensor expected");
  return t.scalar_type() == at::kBFloat16 ? 0 : 1;
}
// rows with unit inner stride
void rows2(const at::Tensor& t, const char* what) { TORCH_CHECK(t.dim() == 2 && t.stride(1) == 1, what, ": [rows, cols] with unit inner stride expected"); }
const float* vecf(const at::Tensor& t, int64_t n, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kFloat && t.is_contiguous() && t.numel() == n, what, ": contiguous fp32 vector of ", n, " expected");
  return t.data_ptr<float>();
}
const float* vecf(const c10::optional<at::Tensor>& t, int64_t n, const char* what) { return t.has_value() ? vecf(*t, n, what) : nullptr; }
template <class I>
const I* veci(const at::Tensor& t, int64_t n, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.scalar_type() == c10::CppTypeToScalarType<I>::value && t.is_contiguous() && t.numel() >= n, what, ": contiguous index vector of at least ",
              n, " expected");
  return t.data_ptr<I>();
}

std::vector<at::Tensor> mix_embed(const at::Tensor& ids, const at::Tensor& emb, const c10::optional<at::Tensor>& w, double eps) {
  const int dt = dt_of(emb, "mix_embed");
  TORCH_CHECK(emb.is_contiguous() && emb.dim() == 2);
  const int64_t rows = ids.numel(), W = emb.size(1);
  const int64_t* ip = veci<int64_t>(ids, rows, "mix_embed ids");
  c10::cuda::CUDAGuard g(emb.device());
  at::Tensor x = at::empty({rows, W}, emb.options().dtype(at::kFloat));
  const bool own = dt == 0 || w.has_value();
  at::Tensor h = own ? at::empty({rows, W}, emb.options()) : x;
  check(prl_mix_embed(ip, emb.data_ptr(), vecf(w, W, "mix_embed w"), x.data_ptr<float>(), own ? h.data_ptr() : nullptr, rows, W, static_cast<float>(eps), dt,
                      cur_stream()), "mix_embed");
  return {x, h};
}

// x += rms(y) * w in place; returns x in y's dtype (x itself when fp32), or the next norm of x when w_next is given
at::Tensor mix_norm_add_(const at::Tensor& y, at::Tensor x, const at::Tensor& w, double eps, const c10::optional<at::Tensor>& w_next) {
  const int dt = dt_of(y, "mix_norm_add");
  rows2(y, "mix_norm_add y");
  CHECK_F32(x);
  TORCH_CHECK(x.is_contiguous() && x.sizes() == y.sizes());
  const int64_t rows = x.size(0), W = x.size(1);
  c10::cuda::CUDAGuard g(y.device());
  const bool own = dt == 0 || w_next.has_value();
  at::Tensor h = own ? at::empty({rows, W}, y.options()) : x;
  check(prl_mix_norm_add(y.data_ptr(), y.stride(0), x.data_ptr<float>(), vecf(w, W, "mix_norm_add w"), vecf(w_next, W, "mix_norm_add w_next"),
                         own ? h.data_ptr() : nullptr, rows, W, static_cast<float>(eps), dt, cur_stream()), "mix_norm_add");
  return h;
}

at::Tensor mix_rms(const at::Tensor& x, const at::Tensor& w, double eps, bool bf16, bool center) {
  CHECK_F32(x);
  TORCH_CHECK(x.is_contiguous() && x.dim() == 2);
  c10::cuda::CUDAGuard g(x.device());
  at::Tensor h = at::empty(x.sizes(), x.options().dtype(bf16 ? at::kBFloat16 : at::kFloat));
  check(prl_mix_rms(x.data_ptr<float>(), vecf(w, x.size(1), "mix_rms w"), h.data_ptr(), x.size(0), x.size(1), static_cast<float>(eps), center, bf16 ? 0 : 1,
                    cur_stream()), "mix_rms");
  return h;
}

at::Tensor mix_gated_norm(const at::Tensor& y, const at::Tensor& z, const at::Tensor& w, int64_t groups, double eps, int64_t gate,
                          const c10::optional<at::Tensor>& to) {
  const int dt = dt_of(y, "mix_gated_norm");
  rows2(y, "mix_gated_norm y"); rows2(z, "mix_gated_norm z");
  TORCH_CHECK(z.scalar_type() == y.scalar_type() && z.sizes() == y.sizes() && groups > 0 && y.size(1) % groups == 0);
  c10::cuda::CUDAGuard g(y.device());
  at::Tensor out = to.has_value() ? *to : at::empty(y.sizes(), y.options());
  TORCH_CHECK(out.is_cuda() && out.scalar_type() == y.scalar_type() && out.sizes() == y.sizes() && out.stride(1) == 1, "mix_gated_norm: out");
  check(prl_mix_gated_norm(y.data_ptr(), y.stride(0), z.data_ptr(), z.stride(0), vecf(w, y.size(1), "mix_gated_norm w"), out.data_ptr(), out.stride(0),
                           y.size(0), groups, y.size(1) / groups, static_cast<float>(eps), static_cast<int>(gate), dt, cur_stream()), "mix_gated_norm");
  return out;
}

// x [T, ch] -> silu(conv(x)); state [slots, taps - 1, ch] is read for what lies before a span and left holding its last inputs
at::Tensor mix_conv(const at::Tensor& x, const at::Tensor& w, const c10::optional<at::Tensor>& bias, at::Tensor state, const at::Tensor& cu, const at::Tensor& start,
                    const at::Tensor& slot, const c10::optional<at::Tensor>& seq_of) {
  const int dt = dt_of(x, "mix_conv");
  rows2(x, "mix_conv x");
  const int64_t T = x.size(0), ch = x.size(1), taps = w.size(0), spans = start.numel();
  TORCH_CHECK(w.dim() == 2 && w.size(1) == ch && state.scalar_type() == x.scalar_type() && state.is_cuda() && state.is_contiguous() && state.dim() == 3 &&
              state.size(1) == taps - 1 && state.size(2) == ch, "mix_conv: shapes");
  TORCH_CHECK(seq_of.has_value() || spans == T, "mix_conv: one token per span without seq_of");
  c10::cuda::CUDAGuard g(x.device());
  at::Tensor out = at::empty({T, ch}, x.options());
  check(prl_mix_conv(x.data_ptr(), x.stride(0), vecf(w, taps * ch, "mix_conv w"), vecf(bias, ch, "mix_conv bias"), state.data_ptr(),
                     veci<int32_t>(cu, spans + 1, "cu"), veci<int32_t>(start, spans, "start"), veci<int64_t>(slot, spans, "slot"),
                     seq_of.has_value() ? veci<int32_t>(*seq_of, T, "seq_of") : nullptr, out.data_ptr(), out.stride(0), ch, taps, T, spans, dt,
                     cur_stream()), "mix_conv");
  return out;
}

// gated linear recurrences over packed spans (mix_scan_): form 0 = token by token, 1 = every span is one token, 2 = chunked (bf16), 3 = chunked on
// tcgen05 where the layout allows, else 2; the last counter element is the error flag; mode 0 = state-space duality, 1 = matrix memory, 2 = gated delta rule, 3 = constant decay, 4 = decay per state row
// (csrc/mixers.cuh)
prl::ScanParams scan_params(int64_t mode, const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, const c10::optional<at::Tensor>& g0, const c10::optional<at::Tensor>& g1,
                            const c10::optional<at::Tensor>& b0, const c10::optional<at::Tensor>& b1, const c10::optional<at::Tensor>& a_log, double qscale,
                            const at::Tensor& S, const at::Tensor& cu, const at::Tensor& start, const at::Tensor& slot, const at::Tensor& counter,
                            const at::Tensor& out) {
  rows2(q, "mix_scan q"); rows2(k, "mix_scan k"); rows2(v, "mix_scan v");
  CHECK_F32(S);
  TORCH_CHECK(mode >= 0 && mode <= 4);
  TORCH_CHECK(S.dim() == 4 && S.is_contiguous());
  const int64_t H = S.size(1), N = S.size(2), V = S.size(3), T = v.size(0), spans = start.numel();
  TORCH_CHECK(q.scalar_type() == v.scalar_type() && k.scalar_type() == v.scalar_type() && q.size(0) == T && k.size(0) == T && v.size(1) == H * V &&
              q.sizes() == k.sizes() && q.size(1) % N == 0 && q.size(1) > 0 && H % (q.size(1) / N) == 0, "mix_scan: shapes");
  TORCH_CHECK(N <= 512, "mix_scan: state rows per head <= 512");
  prl::ScanParams p{};
  p.q = q.data_ptr(); p.k = k.data_ptr(); p.v = v.data_ptr();
  p.ldq = q.stride(0); p.ldk = k.stride(0); p.ldv = v.stride(0);
  p.rep = H / (q.size(1) / N);
  const int64_t gates = mode == 4 ? H * N : H;
  if (mode != 3) {
    TORCH_CHECK(g0.has_value());
    rows2(*g0, "mix_scan g0"); CHECK_F32(*g0);
    TORCH_CHECK(g0->size(0) == T && g0->size(1) == gates, "mix_scan: gates");
    p.g0 = g0->data_ptr<float>(); p.ldg = g0->stride(0);
  }
  p.b0 = vecf(b0, gates, "b0"); p.b1 = vecf(b1, H, "b1"); p.a_log = vecf(a_log, H, "a_log");
  if (mode == 1 || mode == 2) {
    TORCH_CHECK(g1.has_value());
    CHECK_F32(*g1);
    TORCH_CHECK(g1->dim() == 2 && g1->size(0) == T && g1->size(1) == H && g1->stride(1) == 1 && g1->stride(0) == g0->stride(0));
    p.g1 = g1->data_ptr<float>();
  }
  TORCH_CHECK(mode == 1 || mode == 4 || a_log.has_value());
  p.qscale = static_cast<float>(qscale);
  TORCH_CHECK(out.is_cuda() && out.scalar_type() == v.scalar_type() && out.is_contiguous() && out.dim() == 2 && out.size(0) == T && out.size(1) == H * V);
  p.out = out.data_ptr(); p.ldo = H * V;
  p.S = S.data_ptr<float>();
  p.cu = veci<int32_t>(cu, spans + 1, "cu"); p.start = veci<int32_t>(start, spans, "start"); p.slot = veci<int64_t>(slot, spans, "slot");
  veci<int32_t>(counter, spans * H + 1, "counter");
  p.counter = counter.data_ptr<int32_t>();
  p.H = H; p.N = N; p.V = V; p.spans = spans;
  return p;
}

void mix_scan_(int64_t mode, const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, const c10::optional<at::Tensor>& g0, const c10::optional<at::Tensor>& g1,
                     const c10::optional<at::Tensor>& b0, const c10::optional<at::Tensor>& b1, const c10::optional<at::Tensor>& a_log,
                     const c10::optional<at::Tensor>& d_skip, double qscale, double cap, bool raw, at::Tensor S, const c10::optional<at::Tensor>& nst,
                     const c10::optional<at::Tensor>& mst, const at::Tensor& cu, const at::Tensor& start, const at::Tensor& slot, at::Tensor counter,
                     int64_t form, at::Tensor out) {
  const int dt = dt_of(v, "mix_scan");
  prl::ScanParams p = scan_params(mode, q, k, v, g0, g1, b0, b1, a_log, qscale, S, cu, start, slot, counter, out);
  p.d_skip = vecf(d_skip, p.H, "d_skip");
  p.cap = static_cast<float>(cap);
  p.raw = raw;
  TORCH_CHECK(mode != 4 || cap > 0);
  if (mode == 1) {
    TORCH_CHECK(nst.has_value() && mst.has_value());
    CHECK_F32(*nst); CHECK_F32(*mst);
    TORCH_CHECK(nst->is_contiguous() && nst->numel() == S.size(0) * p.H * p.N && mst->is_contiguous() && mst->numel() == S.size(0) * p.H && cap > 0);
    p.nst = nst->data_ptr<float>(); p.mst = mst->data_ptr<float>();
  }
  c10::cuda::CUDAGuard g(v.device());
  TORCH_CHECK(form < 2 || mode < 2 || mode == 3, "mix_scan: no chunked form here");
  if (form == 3 && dt == 0 && prl_mix_chunk_tc_ok(&p)) {
    check(prl_mix_chunk_tc(&p, static_cast<int>(mode), p.counter + counter.numel() - 1, cur_stream()), "mix_chunk_tc");
  } else if (form >= 2) {
    TORCH_CHECK(dt == 0 && prl_mix_chunk_supported(p.N), "mix_scan: the chunked kernel takes bf16 and N <= 256");
    check(prl_mix_chunk(&p, static_cast<int>(mode), cur_stream()), "mix_chunk");
  } else {
    check(prl_mix_scan(&p, static_cast<int>(mode), dt, form == 1, cur_stream()), "mix_scan");
  }
}

bool mix_delta_chunk_ok(const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, const at::Tensor& S) {
  return v.scalar_type() == at::kBFloat16 && prl_mix_delta_ok(q.data_ptr(), q.stride(0), k.data_ptr(), k.stride(0), v.data_ptr(), v.stride(0), S.size(2), S.size(3));
}
// gated delta rule in chunks of 64 tokens (bf16); the last counter element is the error flag
void mix_delta_chunk_(const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, const at::Tensor& g0, const at::Tensor& g1, const c10::optional<at::Tensor>& b0,
                      const at::Tensor& a_log, double qscale, at::Tensor S, const at::Tensor& cu, const at::Tensor& start, const at::Tensor& slot,
                      at::Tensor counter, at::Tensor out) {
  TORCH_CHECK(dt_of(v, "mix_delta_chunk") == 0 && mix_delta_chunk_ok(q, k, v, S), "mix_delta_chunk: layout");
  const prl::ScanParams p = scan_params(2, q, k, v, g0, g1, b0, c10::nullopt, a_log, qscale, S, cu, start, slot, counter, out);
  c10::cuda::CUDAGuard g(v.device());
  const int64_t chunks = prl_mix_delta_chunks(v.size(0), p.spans);
  at::Tensor work = at::empty({chunks * p.H * prl_mix_delta_work_bytes()}, v.options().dtype(at::kByte));
  at::Tensor gates = at::empty({chunks * p.H * prl_mix_delta_gate_floats()}, v.options().dtype(at::kFloat));
  check(prl_mix_delta(&p, v.size(0), chunks, work.data_ptr(), gates.data_ptr<float>(), p.counter + counter.numel() - 1, cur_stream()), "mix_delta_chunk");
}

// gated linear attention in chunks of 64 tokens (bf16); false: the layout is left to mix_scan_.  The last counter element is the error flag
bool mix_gla_chunk_(const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, const at::Tensor& g0, const c10::optional<at::Tensor>& b0, double qscale, double tau,
                    at::Tensor S, const at::Tensor& cu, const at::Tensor& start, const at::Tensor& slot, at::Tensor counter, at::Tensor out) {
  if (dt_of(v, "mix_gla_chunk") != 0) return false;
  prl::ScanParams p = scan_params(4, q, k, v, g0, c10::nullopt, b0, c10::nullopt, c10::nullopt, qscale, S, cu, start, slot, counter, out);
  TORCH_CHECK(tau > 0);
  p.cap = static_cast<float>(tau);
  if (!prl_mix_gla_ok(&p)) return false;
  c10::cuda::CUDAGuard g(v.device());
  const int64_t chunks = prl_mix_gla_chunks(v.size(0), p.spans);
  at::Tensor work = at::empty({chunks * p.H * prl_mix_gla_work_bytes(p.N)}, v.options().dtype(at::kByte));
  at::Tensor keep = at::empty({chunks * p.H * prl_mix_gla_keep_floats(p.N)}, v.options().dtype(at::kFloat));
  check(prl_mix_gla(&p, v.size(0), chunks, work.data_ptr(), keep.data_ptr<float>(), p.counter + counter.numel() - 1, cur_stream()), "mix_gla_chunk");
  return true;
}

// a [T, qr + r + rd] -> (normed query latent [T, qr], packed cache rows [T, r + rd] or empty); cache rows also go to pool[kvslot]
std::vector<at::Tensor> mix_latent_prep(const at::Tensor& a, const at::Tensor& wq, const at::Tensor& wkv, const at::Tensor& freq, const at::Tensor& pos,
                                        const at::Tensor& kvslot, at::Tensor pool, double eps, bool want_entry) {
  const int dt = dt_of(a, "mix_latent_prep");
  rows2(a, "mix_latent_prep a");
  const int64_t T = a.size(0), qr = wq.numel(), r = wkv.numel(), rd = 2 * freq.numel();
  TORCH_CHECK(a.size(1) >= qr + r + rd && pool.scalar_type() == a.scalar_type() && pool.is_cuda() && pool.is_contiguous() && pool.size(-1) == r + rd);
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == at::kDouble && freq.is_contiguous());
  c10::cuda::CUDAGuard g(a.device());
  at::Tensor cq = at::empty({T, qr}, a.options()), en = at::empty({want_entry ? T : 0, r + rd}, a.options());
  check(prl_mix_latent_prep(a.data_ptr(), a.stride(0), qr, r, rd, vecf(wq, qr, "wq"), vecf(wkv, r, "wkv"), freq.data_ptr<double>(),
                            veci<int64_t>(pos, T, "pos"), veci<int64_t>(kvslot, T, "kvslot"), cq.data_ptr(), want_entry ? en.data_ptr() : nullptr,
                            pool.data_ptr(), T, static_cast<float>(eps), dt, cur_stream()), "mix_latent_prep");
  return {cq, en};
}

// q [T, H, dq]: rotate columns [d, d + 2 * freq.numel()) of every head in place
void mix_rope_(at::Tensor q, int64_t d, const at::Tensor& freq, const at::Tensor& pos) {
  const int dt = dt_of(q, "mix_rope");
  TORCH_CHECK(q.dim() == 3 && q.stride(2) == 1 && q.stride(1) == q.size(2) && d + 2 * freq.numel() <= q.size(2));
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == at::kDouble && freq.is_contiguous());
  c10::cuda::CUDAGuard g(q.device());
  check(prl_mix_rope(q.data_ptr(), q.stride(0), q.size(1), q.size(2), d, 2 * freq.numel(), freq.data_ptr<double>(), veci<int64_t>(pos, q.size(0), "pos"),
                     q.size(0), dt, cur_stream()), "mix_rope");
}

// absorbed latent attention: q_lat [H, R, r], q [R, H, dq] (rotated part at column d) over pool rows -> [H, R, r]
at::Tensor mix_latent(const at::Tensor& q_lat, const at::Tensor& q, int64_t d, const at::Tensor& pool, const at::Tensor& table,
                      const c10::optional<at::Tensor>& seq_of, const at::Tensor& kv_len, const c10::optional<at::Tensor>& sink, double scale, int64_t splits,
                      bool tc) {
  const int dt = dt_of(q, "mix_latent");
  TORCH_CHECK(q_lat.dim() == 3 && q_lat.is_contiguous() && q_lat.scalar_type() == q.scalar_type() && q.dim() == 3 && q.stride(2) == 1 &&
              q.stride(1) == q.size(2));
  const int64_t H = q_lat.size(0), R = q_lat.size(1), r = q_lat.size(2), rd = pool.size(-1) - r;
  TORCH_CHECK(q.size(0) == R && q.size(1) == H && rd >= 0 && d + rd <= q.size(2));
  TORCH_CHECK(pool.is_cuda() && pool.is_contiguous() && pool.scalar_type() == q.scalar_type() && (reinterpret_cast<uintptr_t>(pool.data_ptr()) & 15) == 0);
  TORCH_CHECK(table.is_cuda() && table.scalar_type() == at::kInt && table.dim() == 2 && table.stride(1) == 1);
  TORCH_CHECK(seq_of.has_value() || table.size(0) >= R);
  TORCH_CHECK(splits >= 1);
  prl::LatentParams p{};
  p.q_lat = q_lat.data_ptr(); p.q = q.data_ptr(); p.ldq = q.stride(0); p.dq = q.size(2); p.d = d;
  p.pool = pool.data_ptr(); p.table = table.data_ptr<int32_t>(); p.ld_table = table.stride(0);
  p.seq_of = seq_of.has_value() ? veci<int32_t>(*seq_of, R, "seq_of") : nullptr;
  p.kv_len = veci<int32_t>(kv_len, R, "kv_len");
  p.sink = vecf(sink, H, "sink");
  p.H = H; p.R = R; p.r = r; p.rd = rd; p.scale = static_cast<float>(scale);
  p.splits = tc ? splits : 1;
  c10::cuda::CUDAGuard g(q.device());
  at::Tensor out = at::empty({H, R, r}, q.options()), part;
  p.out = out.data_ptr();
  if (p.splits > 1) {
    part = at::empty({H * R * p.splits * (r + 2)}, q.options().dtype(at::kFloat));
    p.part = part.data_ptr<float>();
  }
  check(prl_mix_latent(&p, tc ? 1 : 0, dt, cur_stream()), "mix_latent");
  return out;
}

// rows [queries H x dim | keys G x dim] -> q [T, H, width] (normed, rotated), the same of the keys and the raw keys to the pools
// [pages, G, 16, width] and, when asked for, packed [T, G, width]
std::vector<at::Tensor> mix_qk_prep(const at::Tensor& p, int64_t heads, int64_t dim, const at::Tensor& wq, const at::Tensor& wk, const at::Tensor& freq,
                                    const at::Tensor& pos, const at::Tensor& kvslot, at::Tensor k_pool, at::Tensor v_pool, double eps, bool want_kv) {
  const int dt = dt_of(p, "mix_qk_prep");
  rows2(p, "mix_qk_prep p");
  TORCH_CHECK(k_pool.dim() == 4 && k_pool.size(2) == 16 && k_pool.sizes() == v_pool.sizes());
  for (const at::Tensor& t : {k_pool, v_pool}) TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.scalar_type() == p.scalar_type(), "mix_qk_prep: pools");
  const int64_t T = p.size(0), G = k_pool.size(1), width = k_pool.size(3), rd = 2 * freq.numel();
  TORCH_CHECK(p.size(1) >= (heads + G) * dim && rd <= dim && width >= dim && (width == dim || width % 8 == 0));
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == at::kDouble && freq.is_contiguous());
  c10::cuda::CUDAGuard g(p.device());
  at::Tensor q = at::empty({T, heads, width}, p.options()), k = at::empty({want_kv ? T : 0, G, width}, p.options()), v = at::empty_like(k);
  check(prl_mix_qk_prep(p.data_ptr(), p.stride(0), heads, G, dim, width, rd, vecf(wq, heads * dim, "wq"), vecf(wk, G * dim, "wk"), freq.data_ptr<double>(),
                        veci<int64_t>(pos, T, "pos"), veci<int64_t>(kvslot, T, "kvslot"), q.data_ptr(), want_kv ? k.data_ptr() : nullptr,
                        want_kv ? v.data_ptr() : nullptr, k_pool.data_ptr(), v_pool.data_ptr(), T, static_cast<float>(eps), dt, cur_stream()), "mix_qk_prep");
  return {q, k, v};
}

std::vector<at::Tensor> mix_gather_keys(const at::Tensor& k_pool, const at::Tensor& v_pool, const at::Tensor& rows) {
  for (const at::Tensor& t : {k_pool, v_pool})
    TORCH_CHECK(t.is_cuda() && t.dim() == 4 && t.size(2) == 16 && t.is_contiguous() && t.size(0) == k_pool.size(0) && t.size(1) == k_pool.size(1) &&
                t.scalar_type() == k_pool.scalar_type(), "mix_gather_keys: pools");
  const int64_t n = rows.numel(), G = k_pool.size(1), es = k_pool.element_size();
  c10::cuda::CUDAGuard g(k_pool.device());
  at::Tensor k = at::empty({n, G, k_pool.size(3)}, k_pool.options()), v = at::empty({n, G, v_pool.size(3)}, v_pool.options());
  check(prl_mix_gather_keys(k_pool.data_ptr(), v_pool.data_ptr(), veci<int64_t>(rows, n, "rows"), k.data_ptr(), v.data_ptr(), n, G, k_pool.size(3) * es,
                            v_pool.size(3) * es, cur_stream()), "mix_gather_keys");
  return {k, v};
}

// paged windowed attention, any width: q [R, H, D] -> [R, H, D]
at::Tensor mix_window_attention(const at::Tensor& q, const at::Tensor& k_pool, const at::Tensor& v_pool, const at::Tensor& table,
                                const c10::optional<at::Tensor>& seq_of, const at::Tensor& kv_len, double scale, int64_t window, int64_t keep_first) {
  const int dt = dt_of(q, "mix_window_attention");
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && k_pool.dim() == 4 && k_pool.size(2) == 16 && k_pool.sizes() == v_pool.sizes() && k_pool.size(3) == q.size(2));
  for (const at::Tensor& t : {k_pool, v_pool}) TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.scalar_type() == q.scalar_type(), "mix_window_attention: pools");
  TORCH_CHECK(table.is_cuda() && table.scalar_type() == at::kInt && table.dim() == 2 && table.stride(1) == 1);
  const int64_t R = q.size(0);
  TORCH_CHECK(seq_of.has_value() || table.size(0) >= R);
  TORCH_CHECK(window >= 1 && window <= 0x7fffffff && keep_first >= 0 && keep_first <= 0x7fffffff);
  prl::WindowParams p{};
  p.q = q.data_ptr(); p.k_pool = k_pool.data_ptr(); p.v_pool = v_pool.data_ptr();
  p.table = table.data_ptr<int32_t>(); p.ld_table = table.stride(0);
  p.seq_of = seq_of.has_value() ? veci<int32_t>(*seq_of, R, "seq_of") : nullptr;
  p.kv_len = veci<int32_t>(kv_len, R, "kv_len");
  p.R = R; p.H = q.size(1); p.G = k_pool.size(1); p.D = q.size(2);
  p.window = window; p.keep_first = keep_first; p.scale = static_cast<float>(scale);
  c10::cuda::CUDAGuard g(q.device());
  at::Tensor out = at::empty_like(q);
  p.out = out.data_ptr();
  check(prl_mix_window(&p, dt, cur_stream()), "mix_window_attention");
  return out;
}

at::Tensor gemm_clamped_glu(const at::Tensor& a, const at::Tensor& wgu, double limit, double alpha) {
  CHECK_BF16(a); CHECK_BF16(wgu); CHECK_LASTDIM(a); CHECK_LASTDIM(wgu);
  TORCH_CHECK(a.dim() == 2 && wgu.dim() == 2 && a.size(1) == wgu.size(1) && wgu.size(0) % 256 == 0 && a.size(1) % 8 == 0 && a.stride(0) % 8 == 0 &&
              wgu.stride(0) % 8 == 0, "gemm_clamped_glu: gate / up rows in blocks of 128");
  c10::cuda::CUDAGuard g(a.device());
  at::Tensor h = at::empty({a.size(0), wgu.size(0) / 2}, a.options());
  check(prl_gemm_clamped_glu_bf16(a.data_ptr(), wgu.data_ptr(), h.data_ptr(), a.size(0), wgu.size(0), a.size(1), a.stride(0), wgu.stride(0), h.stride(0),
                                  static_cast<float>(limit), static_cast<float>(alpha), cur_stream()), "gemm_clamped_glu");
  return h;
}
// gu [T, 2 F], gate and up columns in alternating blocks of blk -> [T, F]
at::Tensor mix_clamped_glu(const at::Tensor& gu, int64_t blk, double limit, double alpha) {
  const int dt = dt_of(gu, "mix_clamped_glu");
  TORCH_CHECK(gu.dim() == 2 && gu.is_contiguous() && blk > 0 && gu.size(1) % (2 * blk) == 0);
  c10::cuda::CUDAGuard g(gu.device());
  at::Tensor out = at::empty({gu.size(0), gu.size(1) / 2}, gu.options());
  check(prl_mix_clamped_glu(gu.data_ptr(), out.data_ptr(), gu.size(0), gu.size(1) / 2, blk, static_cast<float>(limit), static_cast<float>(alpha), dt,
                            cur_stream()), "mix_clamped_glu");
  return out;
}

at::Tensor gemm_act(const at::Tensor& a, const at::Tensor& w, bool silu) {
  CHECK_BF16(a); CHECK_BF16(w); CHECK_LASTDIM(a); CHECK_LASTDIM(w);
  TORCH_CHECK(a.dim() == 2 && w.dim() == 2 && a.size(1) == w.size(1) && w.size(0) % 8 == 0 && a.size(1) % 8 == 0 && a.stride(0) % 8 == 0 &&
              w.stride(0) % 8 == 0);
  c10::cuda::CUDAGuard g(a.device());
  at::Tensor h = at::empty({a.size(0), w.size(0)}, a.options());
  check(prl_gemm_gelu_bf16(a.data_ptr(), w.data_ptr(), h.data_ptr(), a.size(0), w.size(0), a.size(1), a.stride(0), w.stride(0), h.stride(0), silu, cur_stream()),
        "gemm_act");
  return h;
}
void mix_act_(at::Tensor x, bool silu) {
  const int dt = dt_of(x, "mix_act");
  TORCH_CHECK(x.is_contiguous());
  c10::cuda::CUDAGuard g(x.device());
  check(prl_mix_gelu(x.data_ptr(), x.numel(), silu, dt, cur_stream()), "mix_act");
}

std::vector<at::Tensor> gemm_swiglu(const at::Tensor& a, const at::Tensor& wgu, bool save_gu) {
  CHECK_BF16(a); CHECK_BF16(wgu); CHECK_LASTDIM(a); CHECK_LASTDIM(wgu);
  const int M = a.size(0), K = a.size(1), N2 = wgu.size(0);
  TORCH_CHECK(wgu.size(1) == K && N2 % 256 == 0 && K % 8 == 0);
  c10::cuda::CUDAGuard g(a.device());
  at::Tensor h = at::empty({M, N2 / 2}, a.options());
  at::Tensor gu = save_gu ? at::empty({M, N2}, a.options()) : at::Tensor();
  check(prl_gemm_swiglu_bf16(a.data_ptr(), wgu.data_ptr(), h.data_ptr(), save_gu ? gu.data_ptr() : nullptr, M, N2, K,
                             a.stride(0), wgu.stride(0), h.stride(0), save_gu ? gu.stride(0) : 0, cur_stream()),
        "gemm_swiglu");
  if (save_gu) return {h, gu};
  return {h};
}

at::Tensor mix_silu_glu(const at::Tensor& gu, int64_t blk) {
  const int dt = dt_of(gu, "mix_silu_glu");
  TORCH_CHECK(gu.dim() == 2 && gu.is_contiguous() && blk > 0 && gu.size(1) % (2 * blk) == 0);
  c10::cuda::CUDAGuard g(gu.device());
  at::Tensor out = at::empty({gu.size(0), gu.size(1) / 2}, gu.options());
  check(prl_mix_silu_glu(gu.data_ptr(), out.data_ptr(), gu.size(0), gu.size(1) / 2, blk, dt, cur_stream()), "mix_silu_glu");
  return out;
}

at::Tensor mix_poly_norm(const at::Tensor& z, const at::Tensor& act, double eps) {
  const int dt = dt_of(z, "mix_poly_norm");
  rows2(z, "mix_poly_norm z");
  c10::cuda::CUDAGuard g(z.device());
  at::Tensor out = at::empty(z.sizes(), z.options());
  check(prl_mix_poly_norm(z.data_ptr(), z.stride(0), vecf(act, 4, "act"), out.data_ptr(), z.size(0), z.size(1), static_cast<float>(eps), dt, cur_stream()),
        "mix_poly_norm");
  return out;
}

// ---------------------------------------------------------------------------------------------- parallel blocks
// convolution of single-token rows at the end of a block kernel (all absent: none)
void block_conv(prl::BlockParams& p, const at::Tensor& like, const c10::optional<at::Tensor>& c1, const c10::optional<at::Tensor>& c2,
                const c10::optional<at::Tensor>& state, const c10::optional<at::Tensor>& start, const c10::optional<at::Tensor>& slot) {
  if (!c1.has_value()) return;
  TORCH_CHECK(state.has_value() && start.has_value() && slot.has_value() && c1->dim() == 2);
  p.taps = c1->size(0);
  p.c1 = vecf(c1, static_cast<int64_t>(p.taps) * p.W, "conv 1");
  p.c2 = vecf(c2, static_cast<int64_t>(p.taps) * p.W, "conv 2");
  TORCH_CHECK(state->is_cuda() && state->scalar_type() == like.scalar_type() && state->is_contiguous() && state->dim() == 3 && state->size(1) == p.taps - 1 &&
              state->size(2) == p.W, "block: convolution state");
  p.state = state->data_ptr();
  p.start = veci<int32_t>(*start, p.R, "start"); p.slot = veci<int64_t>(*slot, p.R, "slot");
}
std::vector<at::Tensor> block_run(prl::BlockParams& p, const at::Tensor& first, const at::Tensor& like, int dt, const c10::optional<at::Tensor>& w_next) {
  at::Tensor h, h2;
  if (w_next.has_value()) {
    p.w_next = vecf(w_next, p.W, "w_next");
    h = at::empty({p.R, p.W}, like.options());
    p.h = h.data_ptr();
    if (p.c2) { h2 = at::empty({p.R, p.W}, like.options()); p.h2 = h2.data_ptr(); }
  } else {
    TORCH_CHECK(!p.c1, "block: a convolution without its norm");
  }
  check(prl_mix_block(&p, dt, cur_stream()), "mix_block");
  return {first, h, h2};
}
// -> (results [slots, T, W] with the embedding in the first, h, h2)
std::vector<at::Tensor> mix_block_embed(const at::Tensor& ids, const at::Tensor& emb, int64_t slots, const at::Tensor& w_norm, double eps, bool center,
                                        const c10::optional<at::Tensor>& c1, const c10::optional<at::Tensor>& c2, const c10::optional<at::Tensor>& state,
                                        const c10::optional<at::Tensor>& start, const c10::optional<at::Tensor>& slot) {
  const int dt = dt_of(emb, "mix_block_embed");
  TORCH_CHECK(emb.is_contiguous() && emb.dim() == 2 && slots >= 1);
  c10::cuda::CUDAGuard g(emb.device());
  prl::BlockParams p{};
  p.R = ids.numel(); p.W = emb.size(1);
  p.ids = veci<int64_t>(ids, p.R, "ids");
  p.emb = emb.data_ptr();
  at::Tensor past = at::empty({slots, p.R, p.W}, emb.options().dtype(at::kFloat));
  p.past = past.data_ptr<float>(); p.stride = past.stride(0);
  p.eps = static_cast<float>(eps); p.center = center;
  block_conv(p, emb, c1, c2, state, start, slot);
  return block_run(p, past, emb, dt, w_norm);
}
// layer i of a stack of parallel blocks -> (x' if wanted, h, h2)
std::vector<at::Tensor> mix_block_add(at::Tensor past, int64_t i, const at::Tensor& y1, const c10::optional<at::Tensor>& y2, const c10::optional<at::Tensor>& rows,
                                      const c10::optional<at::Tensor>& pos, const c10::optional<at::Tensor>& s1, const c10::optional<at::Tensor>& s2,
                                      const c10::optional<at::Tensor>& a_prev, const c10::optional<at::Tensor>& a_cur, const c10::optional<at::Tensor>& w_next,
                                      double eps, bool center, bool want_x, const c10::optional<at::Tensor>& c1, const c10::optional<at::Tensor>& c2,
                                      const c10::optional<at::Tensor>& state, const c10::optional<at::Tensor>& start, const c10::optional<at::Tensor>& slot) {
  const int dt = dt_of(y1, "mix_block_add");
  rows2(y1, "mix_block_add y1");
  CHECK_F32(past);
  prl::BlockParams p{};
  p.R = y1.size(0); p.W = y1.size(1); p.n = i;
  TORCH_CHECK(past.dim() == 3 && past.is_contiguous() && past.size(1) == p.R && past.size(2) == p.W && i >= 0);
  TORCH_CHECK(a_cur.has_value() ? past.size(0) >= i + 2 : !a_prev.has_value(), "mix_block_add: one slot per result");
  c10::cuda::CUDAGuard g(y1.device());
  p.past = past.data_ptr<float>(); p.stride = past.stride(0);
  p.y1 = y1.data_ptr(); p.ld1 = y1.stride(0);
  if (y2.has_value()) {
    rows2(*y2, "mix_block_add y2");
    TORCH_CHECK(y2->scalar_type() == y1.scalar_type() && y2->sizes() == y1.sizes());
    p.y2 = y2->data_ptr(); p.ld2 = y2->stride(0);
  }
  if (rows.has_value()) {
    TORCH_CHECK(pos.has_value() && rows->scalar_type() == y1.scalar_type() && rows->is_contiguous() && rows->dim() == 2 && rows->size(1) == p.W &&
                pos->dim() == 2 && pos->size(0) == p.R);
    p.rows = rows->data_ptr(); p.top = pos->size(1);
    p.pos = veci<int32_t>(*pos, static_cast<int64_t>(p.R) * p.top, "pos");
  }
  p.s1 = vecf(s1, p.W, "s1"); p.s2 = vecf(s2, p.W, "s2");
  p.a_prev = vecf(a_prev, i + 1, "a_prev"); p.a_cur = vecf(a_cur, i + 2, "a_cur");
  p.eps = static_cast<float>(eps); p.center = center;
  at::Tensor x;
  if (want_x) { x = at::empty({p.R, p.W}, past.options()); p.x_out = x.data_ptr<float>(); }
  block_conv(p, y1, c1, c2, state, start, slot);
  return block_run(p, x, y1, dt, w_next);
}

std::vector<at::Tensor> mix_input_conv(const at::Tensor& h, const at::Tensor& w1, const c10::optional<at::Tensor>& w2, at::Tensor state, const at::Tensor& cu,
                                       const at::Tensor& start, const at::Tensor& slot, const c10::optional<at::Tensor>& seq_of) {
  const int dt = dt_of(h, "mix_input_conv");
  rows2(h, "mix_input_conv h");
  const int64_t T = h.size(0), ch = h.size(1), taps = w1.size(0), spans = start.numel();
  TORCH_CHECK(w1.dim() == 2 && w1.size(1) == ch && state.scalar_type() == h.scalar_type() && state.is_cuda() && state.is_contiguous() && state.dim() == 3 &&
              state.size(1) == taps - 1 && state.size(2) == ch, "mix_input_conv: shapes");
  TORCH_CHECK(seq_of.has_value() || spans == T, "mix_input_conv: one token per span without seq_of");
  c10::cuda::CUDAGuard g(h.device());
  at::Tensor o1 = at::empty({T, ch}, h.options()), o2;
  if (w2.has_value()) o2 = at::empty({T, ch}, h.options());
  check(prl_mix_input_conv(h.data_ptr(), h.stride(0), vecf(w1, taps * ch, "w1"), vecf(w2, taps * ch, "w2"), state.data_ptr(), veci<int32_t>(cu, spans + 1, "cu"),
                           veci<int32_t>(start, spans, "start"), veci<int64_t>(slot, spans, "slot"),
                           seq_of.has_value() ? veci<int32_t>(*seq_of, T, "seq_of") : nullptr, o1.data_ptr(), w2.has_value() ? o2.data_ptr() : nullptr, ch, taps,
                           T, spans, dt, cur_stream()), "mix_input_conv");
  return {o1, o2};
}

// ---------------------------------------------------------------------------------------------- residual streams
const float* norm_weight(prl::StreamsParams& p, const c10::optional<at::Tensor>& w) {
  if (!w.has_value()) return nullptr;
  p.w_scalar = w->numel() == 1 && p.W != 1;
  return vecf(w, p.w_scalar ? 1 : p.W, "streams: norm weight");
}
// -> (streams [T, 1, W], h)
std::vector<at::Tensor> mix_streams_embed(const at::Tensor& ids, const at::Tensor& emb, double scale, int64_t streams, const at::Tensor& win, const at::Tensor& w_norm,
                                          double eps) {
  const int dt = dt_of(emb, "mix_streams_embed");
  TORCH_CHECK(emb.is_contiguous() && emb.dim() == 2);
  c10::cuda::CUDAGuard g(emb.device());
  prl::StreamsParams p{};
  p.R = ids.numel(); p.W = emb.size(1); p.S = streams;
  p.ids = veci<int64_t>(ids, p.R, "ids");
  p.emb = emb.data_ptr(); p.scale = static_cast<float>(scale); p.eps = static_cast<float>(eps);
  at::Tensor x = at::empty({p.R, 1, p.W}, emb.options().dtype(at::kFloat)), h = at::empty({p.R, p.W}, emb.options());
  p.x_out = x.data_ptr<float>(); p.row_out = p.W;
  p.win = vecf(win, streams, "win");
  p.w_next = norm_weight(p, w_norm);
  p.h = h.data_ptr();
  check(prl_mix_streams(&p, dt, cur_stream()), "mix_streams_embed");
  return {x, h};
}
// x [T, 1 or streams, W] -> (streams after the sublayer, h), or with `last` (their sum [T, W], h)
std::vector<at::Tensor> mix_streams_add(at::Tensor x, const c10::optional<at::Tensor>& y, const c10::optional<at::Tensor>& bias, const c10::optional<at::Tensor>& rows,
                                        const c10::optional<at::Tensor>& pos, const c10::optional<at::Tensor>& weight, const at::Tensor& mix, const at::Tensor& out,
                                        const c10::optional<at::Tensor>& win, const c10::optional<at::Tensor>& w_next, double eps, bool last) {
  CHECK_F32(x);
  TORCH_CHECK(x.dim() == 3 && x.is_contiguous() && (y.has_value() || rows.has_value()), "mix_streams_add: x [T, streams, W] and something to add");
  const at::Tensor& like = y.has_value() ? *y : *rows;
  const int dt = dt_of(like, "mix_streams_add");
  prl::StreamsParams p{};
  p.R = x.size(0); p.W = x.size(2); p.S = out.numel();
  TORCH_CHECK((x.size(1) == 1 || x.size(1) == p.S) && (last || win.has_value()), "mix_streams_add: streams");
  c10::cuda::CUDAGuard g(x.device());
  p.x_in = x.data_ptr<float>(); p.row_in = x.stride(0); p.stream_in = x.size(1) == 1 ? 0 : p.W;
  if (y.has_value()) {
    rows2(*y, "mix_streams_add y");
    TORCH_CHECK(y->size(0) == p.R && y->size(1) == p.W);
    p.y = y->data_ptr(); p.ldy = y->stride(0);
  }
  p.bias = vecf(bias, p.W, "bias");
  if (rows.has_value()) {
    TORCH_CHECK(pos.has_value() && rows->scalar_type() == like.scalar_type() && rows->is_contiguous() && rows->dim() == 2 && rows->size(1) == p.W &&
                pos->dim() == 2 && pos->size(0) == p.R);
    p.rows = rows->data_ptr(); p.top = pos->size(1);
    p.pos = veci<int32_t>(*pos, static_cast<int64_t>(p.R) * p.top, "pos");
    p.weight = vecf(weight, static_cast<int64_t>(p.R) * p.top, "weight");
  }
  p.mix = vecf(mix, static_cast<int64_t>(p.S) * p.S, "mix"); p.out = vecf(out, p.S, "out"); p.win = vecf(win, p.S, "win");
  p.eps = static_cast<float>(eps);
  p.w_next = norm_weight(p, w_next);
  at::Tensor z, h;
  if (last) {
    z = at::empty({p.R, p.W}, x.options());
    p.sum = z.data_ptr<float>();
  } else {
    z = p.stream_in || p.S == 1 ? x : at::empty({p.R, p.S, p.W}, x.options());
    p.x_out = z.data_ptr<float>(); p.row_out = z.stride(0);
  }
  if (p.w_next) { h = at::empty({p.R, p.W}, like.options()); p.h = h.data_ptr(); }
  check(prl_mix_streams(&p, dt, cur_stream()), "mix_streams_add");
  return {z, h};
}

// ---------------------------------------------------------------------------------------------- selective scan
// the first n_long spans token by token in one CTA per span and channels, the rest as single tokens
at::Tensor mix_selective(const at::Tensor& x, const at::Tensor& dt, const at::Tensor& b, const at::Tensor& c, const at::Tensor& z, const at::Tensor& dt_bias,
                         const at::Tensor& a_neg, const at::Tensor& d_skip, at::Tensor S, const at::Tensor& cu, const at::Tensor& start, const at::Tensor& slot,
                         int64_t n_long) {
  const int d = dt_of(x, "mix_selective");
  for (const at::Tensor& t : {x, b, c, z, dt}) rows2(t, "mix_selective");
  CHECK_F32(dt); CHECK_F32(S);
  const int64_t T = x.size(0), C = x.size(1), N = b.size(1), spans = start.numel();
  for (const at::Tensor& t : {b, c, z}) TORCH_CHECK(t.is_cuda() && t.scalar_type() == x.scalar_type() && t.size(0) == T, "mix_selective: rows");
  TORCH_CHECK(z.size(1) == C && c.size(1) == N && dt.size(0) == T && dt.size(1) == C && S.dim() == 3 && S.is_contiguous() && S.size(1) == C && S.size(2) == N &&
              n_long >= 0 && n_long <= spans, "mix_selective: shapes");
  prl::SelectiveParams p{};
  p.x = x.data_ptr(); p.z = z.data_ptr(); p.b = b.data_ptr(); p.c = c.data_ptr();
  p.ldx = x.stride(0); p.ldz = z.stride(0); p.ldb = b.stride(0); p.ldc = c.stride(0);
  p.dt = dt.data_ptr<float>(); p.ldd = dt.stride(0);
  p.dt_bias = vecf(dt_bias, C, "dt_bias"); p.d_skip = vecf(d_skip, C, "d_skip"); p.a_neg = vecf(a_neg, C * N, "a_neg");
  c10::cuda::CUDAGuard g(x.device());
  at::Tensor out = at::empty({T, C}, x.options());
  p.out = out.data_ptr(); p.ldo = C;
  p.S = S.data_ptr<float>();
  p.cu = veci<int32_t>(cu, spans + 1, "cu"); p.start = veci<int32_t>(start, spans, "start"); p.slot = veci<int64_t>(slot, spans, "slot");
  p.C = C; p.N = N;
  p.spans = n_long;
  check(prl_mix_selective(&p, d, 0, cur_stream()), "mix_selective");
  p.cu += n_long; p.start += n_long; p.slot += n_long;
  p.spans = spans - n_long;
  check(prl_mix_selective(&p, d, 1, cur_stream()), "mix_selective step");
  return out;
}

// ---------------------------------------------------------------------------------------------- attention with rotated values and a sink
// rows [queries H x D | keys G x D | values G x V] -> q [T, H, kw], pools, and packed keys / values when asked for
std::vector<at::Tensor> mix_turn_prep(const at::Tensor& p, const at::Tensor& bias, int64_t heads, int64_t dim, int64_t vdim, const at::Tensor& freq,
                                      const at::Tensor& vfreq, const at::Tensor& pos, const at::Tensor& kvslot, at::Tensor k_pool, at::Tensor v_pool, double eps,
                                      bool want_kv) {
  const int dt = dt_of(p, "mix_turn_prep");
  rows2(p, "mix_turn_prep p");
  for (const at::Tensor& t : {k_pool, v_pool})
    TORCH_CHECK(t.is_cuda() && t.dim() == 4 && t.size(2) == 16 && t.is_contiguous() && t.scalar_type() == p.scalar_type() && t.size(0) == k_pool.size(0) &&
                t.size(1) == k_pool.size(1), "mix_turn_prep: pools");
  for (const at::Tensor& t : {freq, vfreq}) TORCH_CHECK(t.is_cuda() && t.scalar_type() == at::kDouble && t.is_contiguous());
  const int64_t T = p.size(0), G = k_pool.size(1), kw = k_pool.size(3), vw = v_pool.size(3), rd = 2 * freq.numel(), cols = (heads + G) * dim + G * vdim;
  TORCH_CHECK(p.size(1) >= cols && G >= 1 && heads % G == 0 && 2 * vfreq.numel() == vdim, "mix_turn_prep: sizes");
  c10::cuda::CUDAGuard g(p.device());
  at::Tensor q = at::empty({T, heads, kw}, p.options()), k = at::empty({want_kv ? T : 0, G, kw}, p.options()), v = at::empty({want_kv ? T : 0, G, vw}, p.options());
  check(prl_mix_turn_rows(p.data_ptr(), p.stride(0), vecf(bias, cols, "bias"), freq.data_ptr<double>(), vfreq.data_ptr<double>(), veci<int64_t>(pos, T, "pos"),
                          veci<int64_t>(kvslot, T, "kvslot"), q.data_ptr(), want_kv ? k.data_ptr() : nullptr, want_kv ? v.data_ptr() : nullptr, k_pool.data_ptr(),
                          v_pool.data_ptr(), T, heads, G, dim, vdim, rd, kw, vw, static_cast<float>(eps), dt, cur_stream()), "mix_turn_prep");
  return {q, k, v};
}
// o [T, H, vw] turned back, times scale * sigmoid(gate) -> out [T, H * vdim]
void mix_turn_back(const at::Tensor& o, const at::Tensor& gate, const at::Tensor& vfreq, const at::Tensor& pos, double scale, at::Tensor out) {
  const int dt = dt_of(o, "mix_turn_back");
  rows2(gate, "mix_turn_back gate"); rows2(out, "mix_turn_back out");
  const int64_t T = o.size(0), H = o.size(1), V = 2 * vfreq.numel();
  TORCH_CHECK(o.dim() == 3 && o.is_contiguous() && o.size(2) >= V && gate.scalar_type() == o.scalar_type() && out.scalar_type() == o.scalar_type() && out.is_cuda() &&
              gate.size(0) == T && gate.size(1) == H * V && out.size(0) == T && out.size(1) == H * V, "mix_turn_back: shapes");
  TORCH_CHECK(vfreq.is_cuda() && vfreq.scalar_type() == at::kDouble && vfreq.is_contiguous());
  c10::cuda::CUDAGuard g(o.device());
  check(prl_mix_turn_back(o.data_ptr(), gate.data_ptr(), gate.stride(0), vfreq.data_ptr<double>(), veci<int64_t>(pos, T, "pos"), static_cast<float>(scale),
                          out.data_ptr(), out.stride(0), T, H, V, o.size(2), dt, cur_stream()), "mix_turn_back");
}
void sink_pools(const at::Tensor& q, const at::Tensor& k_pool, const at::Tensor& v_pool, const at::Tensor& table, const char* what) {
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && k_pool.dim() == 4 && k_pool.size(3) == q.size(2), what, ": q [rows, heads, key width]");
  for (const at::Tensor& t : {k_pool, v_pool})
    TORCH_CHECK(t.is_cuda() && t.dim() == 4 && t.size(2) == 16 && t.is_contiguous() && t.scalar_type() == q.scalar_type() && t.size(0) == k_pool.size(0) &&
                t.size(1) == k_pool.size(1), what, ": pools");
  TORCH_CHECK(k_pool.size(1) >= 1 && q.size(1) % k_pool.size(1) == 0, what, ": heads");
  TORCH_CHECK(table.is_cuda() && table.scalar_type() == at::kInt && table.dim() == 2 && table.stride(1) == 1, what, ": table");
}
// paged, any widths: q [R, H, D] -> [R, H, V]
at::Tensor mix_sink_attention(const at::Tensor& q, const at::Tensor& k_pool, const at::Tensor& v_pool, const at::Tensor& table, const c10::optional<at::Tensor>& seq_of,
                              const at::Tensor& kv_len, double scale, const c10::optional<at::Tensor>& sink) {
  const int dt = dt_of(q, "mix_sink_attention");
  sink_pools(q, k_pool, v_pool, table, "mix_sink_attention");
  const int64_t R = q.size(0);
  TORCH_CHECK(seq_of.has_value() || table.size(0) >= R);
  prl::SinkParams p{};
  p.q = q.data_ptr(); p.k_pool = k_pool.data_ptr(); p.v_pool = v_pool.data_ptr();
  p.table = table.data_ptr<int32_t>(); p.ld_table = table.stride(0);
  p.seq_of = seq_of.has_value() ? veci<int32_t>(*seq_of, R, "seq_of") : nullptr;
  p.kv_len = veci<int32_t>(kv_len, R, "kv_len");
  p.R = R; p.H = q.size(1); p.G = k_pool.size(1); p.D = q.size(2); p.V = v_pool.size(3);
  p.sink = vecf(sink, p.H, "sink");
  p.scale = static_cast<float>(scale);
  c10::cuda::CUDAGuard g(q.device());
  at::Tensor out = at::empty({R, p.H, p.V}, q.options());
  p.out = out.data_ptr();
  check(prl_mix_sink(&p, dt, cur_stream()), "mix_sink_attention");
  return out;
}
// single tokens on the tensor cores (bf16): widths and heads of prl_sink_decode
at::Tensor sink_decode(const at::Tensor& q, const at::Tensor& k_pool, const at::Tensor& v_pool, const at::Tensor& table, const at::Tensor& kv_len, double scale,
                       int64_t splits, const at::Tensor& sink) {
  CHECK_BF16(q);
  sink_pools(q, k_pool, v_pool, table, "sink_decode");
  const int64_t R = q.size(0), H = q.size(1), G = k_pool.size(1), kw = q.size(2), vw = v_pool.size(3);
  TORCH_CHECK(table.size(0) >= R && splits >= 1, "sink_decode: sizes");
  c10::cuda::CUDAGuard g(q.device());
  at::Tensor out = at::empty({R, H, vw}, q.options());
  at::Tensor work = at::empty({prl_paged_decode_workspace_floats(R, H, vw, splits)}, q.options().dtype(at::kFloat));
  check(prl_sink_decode(q.data_ptr(), k_pool.data_ptr(), v_pool.data_ptr(), table.data_ptr<int32_t>(), table.stride(0), veci<int32_t>(kv_len, R, "kv_len"), R, H, G,
                        kw, vw, static_cast<float>(scale), splits, vecf(sink, H, "sink"), work.data_ptr<float>(), out.data_ptr(), cur_stream()), "sink_decode");
  return out;
}

// ---------------------------------------------------------------------------------------------- experts
// logits [T, E] -> (experts [T, top], scores, ranks, plan); counter: >= E + 1 zeros, left zero
std::vector<at::Tensor> mix_route(const at::Tensor& logits, int64_t top, at::Tensor counter, bool softmax) {
  CHECK_F32(logits);
  rows2(logits, "mix_route logits");
  const int64_t T = logits.size(0), E = logits.size(1);
  TORCH_CHECK(top >= 1 && top <= E && T * top < 0x7fffffff);
  veci<int32_t>(counter, E + 1, "counter");
  c10::cuda::CUDAGuard g(logits.device());
  const auto i32 = logits.options().dtype(at::kInt);
  at::Tensor pick = at::empty({T, top}, i32), score = at::empty({T, top}, logits.options()), rank = at::empty({T, top}, i32);
  at::Tensor plan = at::empty({1 + E + prl_mix_route_tiles(T * top, E)}, i32);
  check(prl_mix_route(logits.data_ptr<float>(), logits.stride(0), T, E, top, pick.data_ptr<int32_t>(), score.data_ptr<float>(), rank.data_ptr<int32_t>(),
                      counter.data_ptr<int32_t>(), plan.data_ptr<int32_t>(), softmax, cur_stream()), "mix_route");
  return {pick, score, rank, plan};
}
// -> (rows in the experts' order [tiles * 128, W], place of every (token, choice))
std::vector<at::Tensor> mix_expert_rows(const at::Tensor& h, const at::Tensor& pick, const c10::optional<at::Tensor>& score, const at::Tensor& rank, const at::Tensor& plan,
                                        int64_t experts) {
  const int dt = dt_of(h, "mix_expert_rows");
  rows2(h, "mix_expert_rows h");
  const int64_t T = h.size(0), W = h.size(1), top = pick.size(1), tiles = prl_mix_route_tiles(T * top, experts);
  c10::cuda::CUDAGuard g(h.device());
  at::Tensor rows = at::empty({tiles * 128, W}, h.options()), pos = at::empty({T, top}, pick.options());
  check(prl_mix_expert_rows(h.data_ptr(), h.stride(0), veci<int32_t>(pick, T * top, "pick"), vecf(score, T * top, "score"), veci<int32_t>(rank, T * top, "rank"),
                            veci<int32_t>(plan, 1 + experts + tiles, "plan"), rows.data_ptr(), pos.data_ptr<int32_t>(), T, top, W, dt, cur_stream()),
        "mix_expert_rows");
  return {rows, pos};
}
// rows [tiles * 128, K] x w [experts * N, K]
at::Tensor mix_expert_gemm(const at::Tensor& x, const at::Tensor& w, const at::Tensor& plan, int64_t experts) {
  const int dt = dt_of(x, "mix_expert_gemm");
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && w.is_cuda() && w.dim() == 2 && w.is_contiguous() && w.scalar_type() == x.scalar_type() && w.size(1) == x.size(1) &&
              x.size(0) % 128 == 0 && experts >= 1 && w.size(0) % experts == 0, "mix_expert_gemm: shapes");
  const int64_t tiles = x.size(0) / 128, N = w.size(0) / experts;
  c10::cuda::CUDAGuard g(x.device());
  at::Tensor out = at::empty({x.size(0), N}, x.options());
  check(prl_mix_expert_gemm(x.data_ptr(), w.data_ptr(), veci<int32_t>(plan, 1 + experts + tiles, "plan"), out.data_ptr(), tiles, experts, N, x.size(1), dt,
                            cur_stream()), "mix_expert_gemm");
  return out;
}
// the same on tcgen05 (bf16); glu: w holds gate and up rows in blocks of 128, the result is silu(gate) * up (1) or the clamped gate (2)
at::Tensor gemm_experts(const at::Tensor& x, const at::Tensor& w, const at::Tensor& plan, int64_t experts, int64_t glu, double limit, double alpha) {
  CHECK_BF16(x); CHECK_BF16(w);
  TORCH_CHECK(x.dim() == 2 && x.is_contiguous() && w.dim() == 2 && w.is_contiguous() && w.size(1) == x.size(1) && x.size(0) % 128 == 0 && experts >= 1 &&
              w.size(0) % experts == 0 && x.size(1) % 8 == 0, "gemm_experts: shapes");
  const int64_t tiles = x.size(0) / 128, N = w.size(0) / experts;
  c10::cuda::CUDAGuard g(x.device());
  at::Tensor out = at::empty({x.size(0), glu ? N / 2 : N}, x.options());
  check(prl_gemm_experts_bf16(x.data_ptr(), w.data_ptr(), out.data_ptr(), veci<int32_t>(plan, 1 + experts + tiles, "plan"), tiles, experts, N, x.size(1), glu,
                              static_cast<float>(limit), static_cast<float>(alpha), cur_stream()), "gemm_experts");
  return out;
}

// ---------------------------------------------------------------------------------------------- differential attention
// rows [queries H x 2 x D | keys G x 2 x D | values G x V] -> q [T, 2 H, qw], pools, and packed keys / values when asked for
std::vector<at::Tensor> mix_map_prep(const at::Tensor& p, const at::Tensor& bias, int64_t heads, int64_t dim, int64_t vdim, const at::Tensor& wq,
                                     const at::Tensor& wk, const at::Tensor& freq, const at::Tensor& pos, const at::Tensor& kvslot, at::Tensor k_pool,
                                     at::Tensor v_pool, double eps, bool want_kv, int64_t qw) {
  const int dt = dt_of(p, "mix_map_prep");
  rows2(p, "mix_map_prep p");
  for (const at::Tensor& t : {k_pool, v_pool})
    TORCH_CHECK(t.is_cuda() && t.dim() == 4 && t.size(2) == 16 && t.is_contiguous() && t.scalar_type() == p.scalar_type() && t.size(0) == k_pool.size(0) &&
                t.size(1) == k_pool.size(1), "mix_map_prep: pools");
  const int64_t T = p.size(0), G = k_pool.size(1), kw = k_pool.size(3) / 2, vw = v_pool.size(3), rd = 2 * freq.numel(), cols = 2 * (heads + G) * dim + G * vdim;
  TORCH_CHECK(p.size(1) >= cols && k_pool.size(3) == 2 * kw && G >= 1 && heads % G == 0);
  TORCH_CHECK(freq.is_cuda() && freq.scalar_type() == at::kDouble && freq.is_contiguous());
  c10::cuda::CUDAGuard g(p.device());
  at::Tensor q = at::empty({T, 2 * heads, qw}, p.options()), k = at::empty({want_kv ? T : 0, G, 2 * kw}, p.options()),
             v = at::empty({want_kv ? T : 0, G, vw}, p.options());
  check(prl_mix_map_rows(p.data_ptr(), p.stride(0), vecf(bias, cols, "bias"), vecf(wq, dim, "wq"), vecf(wk, dim, "wk"), freq.data_ptr<double>(),
                         veci<int64_t>(pos, T, "pos"), veci<int64_t>(kvslot, T, "kvslot"), q.data_ptr(), want_kv ? k.data_ptr() : nullptr,
                         want_kv ? v.data_ptr() : nullptr, k_pool.data_ptr(), v_pool.data_ptr(), T, heads, G, dim, vdim, rd, qw, kw, vw, static_cast<float>(eps), dt,
                         cur_stream()), "mix_map_prep");
  return {q, k, v};
}
void map_pools(const at::Tensor& q, const at::Tensor& k_pool, const at::Tensor& v_pool, const at::Tensor& table, int64_t window, const char* what) {
  TORCH_CHECK(q.dim() == 3 && q.is_contiguous() && q.size(1) % 2 == 0, what, ": q [rows, 2 heads, width]");
  for (const at::Tensor& t : {k_pool, v_pool})
    TORCH_CHECK(t.is_cuda() && t.dim() == 4 && t.size(2) == 16 && t.is_contiguous() && t.scalar_type() == q.scalar_type() && t.size(0) == k_pool.size(0) &&
                t.size(1) == k_pool.size(1), what, ": pools");
  TORCH_CHECK(k_pool.size(3) % 2 == 0 && k_pool.size(1) >= 1 && (q.size(1) / 2) % k_pool.size(1) == 0, what, ": heads");
  TORCH_CHECK(q.size(2) == k_pool.size(3) / 2 || q.size(2) == k_pool.size(3), what, ": query width");
  TORCH_CHECK(table.is_cuda() && table.scalar_type() == at::kInt && table.dim() == 2 && table.stride(1) == 1, what, ": table");
  TORCH_CHECK(window >= 1 && window <= 0x7fffffff, what, ": window");
}
at::Tensor mix_map_attention(const at::Tensor& q, const at::Tensor& k_pool, const at::Tensor& v_pool, const at::Tensor& table,
                             const c10::optional<at::Tensor>& seq_of, const at::Tensor& kv_len, double scale, int64_t window, const at::Tensor& lam, double diff,
                             double eps, int64_t vdim, int64_t dim) {
  const int dt = dt_of(q, "mix_map_attention");
  map_pools(q, k_pool, v_pool, table, window, "mix_map_attention");
  prl::MapParams p{};
  p.R = q.size(0); p.H = q.size(1) / 2; p.G = k_pool.size(1); p.qw = q.size(2); p.kw = k_pool.size(3) / 2; p.vw = v_pool.size(3); p.D = dim; p.V = vdim;
  TORCH_CHECK(dim >= 1 && dim <= p.kw && vdim >= 1 && vdim <= p.vw && (seq_of.has_value() || table.size(0) >= p.R));
  p.q = q.data_ptr(); p.k_pool = k_pool.data_ptr(); p.v_pool = v_pool.data_ptr();
  p.table = table.data_ptr<int32_t>(); p.ld_table = table.stride(0);
  p.seq_of = seq_of.has_value() ? veci<int32_t>(*seq_of, p.R, "seq_of") : nullptr;
  p.kv_len = veci<int32_t>(kv_len, p.R, "kv_len");
  p.lam = vecf(lam, 1, "lam");
  p.window = window; p.scale = static_cast<float>(scale); p.keep = static_cast<float>(1.0 - diff); p.eps = static_cast<float>(eps);
  c10::cuda::CUDAGuard g(q.device());
  at::Tensor out = at::empty({p.R, p.H * vdim}, q.options());
  p.out = out.data_ptr();
  check(prl_mix_map_attention(&p, dt, cur_stream()), "mix_map_attention");
  return out;
}
at::Tensor map_decode(const at::Tensor& q, const at::Tensor& k_pool, const at::Tensor& v_pool, const at::Tensor& table, const at::Tensor& kv_len, double scale,
                      int64_t splits, int64_t window, const at::Tensor& lam, double diff, double eps, int64_t vdim) {
  CHECK_BF16(q);
  map_pools(q, k_pool, v_pool, table, window, "map_decode");
  const int64_t R = q.size(0), H = q.size(1) / 2, G = k_pool.size(1), kw = k_pool.size(3) / 2, vw = v_pool.size(3);
  TORCH_CHECK(prl_map_decode_ok(kw, vw, H / G) && q.size(2) == 64 && table.size(0) >= R && splits >= 1, "map_decode: sizes");
  c10::cuda::CUDAGuard g(q.device());
  at::Tensor out = at::empty({R, H * vdim}, q.options());
  at::Tensor work = at::empty({prl_paged_decode_workspace_floats(R, 2 * H, vw, splits)}, q.options().dtype(at::kFloat));
  check(prl_map_decode(q.data_ptr(), k_pool.data_ptr(), v_pool.data_ptr(), table.data_ptr<int32_t>(), table.stride(0), veci<int32_t>(kv_len, R, "kv_len"), R, H, G,
                       kw, vw, vdim, static_cast<float>(scale), splits, window, vecf(lam, 1, "lam"), static_cast<float>(1.0 - diff), static_cast<float>(eps),
                       work.data_ptr<float>(), out.data_ptr(), cur_stream()), "map_decode");
  return out;
}
at::Tensor map_attn_fwd(const at::Tensor& q, const at::Tensor& k, const at::Tensor& v, const at::Tensor& cu_q, const at::Tensor& cu_k, double scale, int64_t window,
                        const at::Tensor& lam, double diff, double eps, int64_t vdim) {
  CHECK_BF16(q); CHECK_BF16(k); CHECK_BF16(v);
  const int64_t dk = q.size(-1), G = k.size(1), dv = v.size(-1);
  TORCH_CHECK(q.dim() == 3 && k.dim() == 3 && v.dim() == 3 && q.is_contiguous() && k.is_contiguous() && v.is_contiguous() && q.size(1) % 2 == 0 && G >= 1 &&
              (q.size(1) / 2) % G == 0 && v.size(1) == G && v.size(0) == k.size(0) && (k.size(2) == 2 * dk || (k.size(2) == 64 && dk == 64)), "map_attn_fwd: shapes");
  for (const at::Tensor& t : {q, k, v}) TORCH_CHECK((reinterpret_cast<uintptr_t>(t.data_ptr()) & 15) == 0, "map_attn_fwd: 16-byte aligned operands");
  TORCH_CHECK(window >= 1 && window <= 0x7fffffff);
  const int Tq = q.size(0), B = cu_q.numel() - 1;
  veci<int32_t>(cu_q, B + 1, "cu_q"); veci<int32_t>(cu_k, B + 1, "cu_k");
  c10::cuda::CUDAGuard g(q.device());
  at::Tensor out = at::empty({Tq, q.size(1) / 2 * vdim}, q.options());
  check(prl_map_attn_fwd(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), cu_q.data_ptr<int32_t>(), cu_k.data_ptr<int32_t>(), B, Tq, k.size(0),
                         q.size(1) / 2, G, dk, dv, vdim, k.size(2) == dk, static_cast<float>(scale), window, vecf(lam, 1, "lam"), static_cast<float>(1.0 - diff),
                         static_cast<float>(eps), Tq / 128 + B, cur_stream()), "map_attn_fwd");
  return out;
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  py::class_<prl::EngineScheduler>(m, "EngineScheduler")
      .def(py::init<prl::KvPageManager*, int64_t, int64_t, bool>(), py::arg("kv"), py::arg("max_num_seqs"), py::arg("page_size"),
           py::arg("prefix_cache"), py::keep_alive<1, 2>())
      .def("add", &prl::EngineScheduler::add, py::arg("prompt"), py::arg("max_new"), py::arg("group"), py::arg("cacheable"))
      .def("remove_waiting", &prl::EngineScheduler::remove_waiting)
      .def("num_waiting", &prl::EngineScheduler::num_waiting)
      .def("num_free_slots", &prl::EngineScheduler::num_free_slots)
      .def("num_live", &prl::EngineScheduler::num_live)
      .def("admit", &prl::EngineScheduler::admit)
      .def("info", [](const prl::EngineScheduler& s, int64_t h) {        // (slot, blocks, shared_prefix_blocks, cached_tokens, donor)
        const prl::SchedRequest& r = s.get(h);
        return py::make_tuple(r.slot, r.blocks, r.shared_prefix_blocks, r.cached_tokens, r.donor);
      })
      .def("prefill_arrays", [](const prl::EngineScheduler& s, const std::vector<std::tuple<int64_t, int64_t, int64_t>>& spans, bool gather) {
        const prl::PrefillArrays a = s.prefill_arrays(spans, gather);
        return py::make_tuple(vec_i64(a.ids), vec_i64(a.pos), vec_i64(a.slots), vec_i64(a.lens), vec_i64(a.g_blk), vec_i64(a.g_off), vec_i64(a.klens));
      })
      .def("block_rows", [](const prl::EngineScheduler& s, const std::vector<int64_t>& handles, int64_t width) {
        const std::vector<int32_t> rows = s.block_rows(handles, width);
        return at::tensor(c10::ArrayRef<int32_t>(rows.data(), rows.size()), at::TensorOptions().dtype(at::kInt))
            .reshape({static_cast<int64_t>(handles.size()), width});
      })
      .def("open", &prl::EngineScheduler::open, py::arg("tokens"))
      .def("feed", &prl::EngineScheduler::feed, py::arg("handle"), py::arg("tokens"))
      .def("move_slots", &prl::EngineScheduler::move_slots)
      .def("free_slots", &prl::EngineScheduler::free_slots)
      .def("finish", &prl::EngineScheduler::finish, py::arg("handle"), py::arg("tokens"), py::arg("to_cache"));
  py::class_<prl::KvPageManager>(m, "KvPageManager")
      .def(py::init<int64_t, int64_t>(), py::arg("num_blocks"), py::arg("page_size"))
      .def_property_readonly("num_blocks", &prl::KvPageManager::num_blocks)
      .def("available", &prl::KvPageManager::available)
      .def("ref", &prl::KvPageManager::ref)
      .def("alloc", &prl::KvPageManager::alloc)
      .def("share", &prl::KvPageManager::share)
      .def("release", &prl::KvPageManager::release)
      .def("page_keys", &prl::KvPageManager::page_keys)
      .def("match", &prl::KvPageManager::match)
      .def("insert", &prl::KvPageManager::insert)
      .def("evict", &prl::KvPageManager::evict)
      .def("flush", &prl::KvPageManager::flush)
      .def("cached_pages", &prl::KvPageManager::cached_pages)
      .def_property_readonly("hits", &prl::KvPageManager::hits)
      .def_property_readonly("misses", &prl::KvPageManager::misses);
  m.def("gemm_bf16", &gemm_bf16, py::arg("a"), py::arg("b"), py::arg("residual") = py::none(),
        py::arg("out") = py::none(), py::arg("force_bn") = 0);
  m.def("attn_fwd", &attn_fwd, py::arg("q"), py::arg("k"), py::arg("v"), py::arg("cu_q"), py::arg("cu_k"), py::arg("sm_scale"),
        py::arg("causal") = true, py::arg("want_lse") = true, py::arg("dbg") = py::none(), py::arg("sink") = py::none(), py::arg("window") = 0,
        py::arg("keep_first") = 0);
  m.def("paged_decode", &paged_decode, py::arg("q"), py::arg("k_cache"), py::arg("v_cache"), py::arg("block_table"),
        py::arg("seq_lens"), py::arg("nq"), py::arg("nkv"), py::arg("d"), py::arg("sm_scale"), py::arg("splits") = 1,
        py::arg("out") = py::none(), py::arg("window") = 0, py::arg("keep_first") = 0);
  m.def("sample", &sample);
  m.def("sample_topk_topp", &sample_topk_topp);
  m.def("mix_embed", &mix_embed);
  m.def("mix_norm_add_", &mix_norm_add_);
  m.def("mix_rms", &mix_rms);
  m.def("mix_gated_norm", &mix_gated_norm);
  m.def("mix_conv", &mix_conv);
  m.def("mix_scan_", &mix_scan_);
  m.def("mix_latent_prep", &mix_latent_prep);
  m.def("mix_rope_", &mix_rope_);
  m.def("mix_latent", &mix_latent);
  m.def("mix_delta_chunk_ok", &mix_delta_chunk_ok);
  m.def("mix_delta_chunk_", &mix_delta_chunk_);
  m.def("mix_gla_chunk_", &mix_gla_chunk_);
  m.def("mix_qk_prep", &mix_qk_prep);
  m.def("mix_gather_keys", &mix_gather_keys);
  m.def("mix_window_attention", &mix_window_attention);
  m.def("gemm_clamped_glu", &gemm_clamped_glu);
  m.def("mix_clamped_glu", &mix_clamped_glu);
  m.def("gemm_gelu", [](const at::Tensor& a, const at::Tensor& w) { return gemm_act(a, w, false); });
  m.def("gemm_silu", [](const at::Tensor& a, const at::Tensor& w) { return gemm_act(a, w, true); });
  m.def("mix_gelu_", [](at::Tensor x) { mix_act_(x, false); });
  m.def("mix_silu_", [](at::Tensor x) { mix_act_(x, true); });
  m.def("mix_streams_embed", &mix_streams_embed);
  m.def("mix_streams_add", &mix_streams_add);
  m.def("mix_selective", &mix_selective);
  m.def("mix_turn_prep", &mix_turn_prep);
  m.def("mix_turn_back", &mix_turn_back);
  m.def("mix_sink_attention", &mix_sink_attention);
  m.def("sink_decode", &sink_decode);
  m.def("gemm_swiglu", &gemm_swiglu);
  m.def("mix_silu_glu", &mix_silu_glu);
  m.def("mix_poly_norm", &mix_poly_norm);
  m.def("mix_block_embed", &mix_block_embed);
  m.def("mix_block_add", &mix_block_add);
  m.def("mix_input_conv", &mix_input_conv);
  m.def("mix_route", &mix_route, py::arg("logits"), py::arg("top"), py::arg("counter"), py::arg("softmax") = false);
  m.def("mix_expert_rows", &mix_expert_rows);
  m.def("mix_expert_gemm", &mix_expert_gemm);
  m.def("gemm_experts", &gemm_experts, py::arg("x"), py::arg("w"), py::arg("plan"), py::arg("experts"), py::arg("glu"), py::arg("limit") = 0.0,
        py::arg("alpha") = 0.0);
  m.def("mix_map_prep", &mix_map_prep);
  m.def("mix_map_attention", &mix_map_attention);
  m.def("map_attn_fwd", &map_attn_fwd);
  m.def("map_decode", &map_decode);
  m.def("map_decode_ok", [](int64_t kw, int64_t vw, int64_t rep) { return prl_map_decode_ok(static_cast<int>(kw), static_cast<int>(vw), static_cast<int>(rep)) != 0; });
  m.def("mix_chunk_supported", [](int64_t n) { return prl_mix_chunk_supported(static_cast<int>(n)) != 0; });
  m.def("mix_latent_tc_ok", [](int64_t r, int64_t rd) { return prl_mix_latent_tc_ok(static_cast<int>(r), static_cast<int>(rd)) != 0; });
}

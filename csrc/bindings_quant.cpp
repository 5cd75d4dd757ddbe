// Python bindings of the quantised-weight kernels (torch extension `oxb_quant`): GGUF block GEMVs and
// dequantisers, block-scaled fp8 GEMM, activation quantisers. Loaded when a model with such weights is.
#include <ATen/cuda/CUDAContext.h>
#include <c10/cuda/CUDAGuard.h>
#include <cuda.h>
#include <cuda_runtime.h>
#include <pybind11/stl.h>
#include <torch/extension.h>

#include <string>
#include <vector>

#include "common/device_info.h"
#include "common/tma_host.h"
#include "kernels/gemm_bf16.cuh"
#include "kernels/gemm_fp8_block.cuh"
#include "kernels/quant_ops.cuh"

namespace py = pybind11;
using torch::Tensor;

namespace {

cudaStream_t cur_stream() { return at::cuda::getCurrentCUDAStream().stream(); }

void check_launch(const char* what) {
  cudaError_t e = cudaGetLastError();
  TORCH_CHECK(e == cudaSuccess, "oxb: launch of ", what, " failed: ", cudaGetErrorString(e));
}

const __nv_bfloat16* bf16_ptr(const c10::optional<Tensor>& t) {
  if (!t.has_value() || !t->defined()) return nullptr;
  TORCH_CHECK(t->scalar_type() == torch::kBFloat16 && t->is_cuda(), "expected a CUDA bf16 tensor");
  return reinterpret_cast<const __nv_bfloat16*>(t->data_ptr());
}
template <typename T>
T* opt_ptr(const c10::optional<Tensor>& t) {
  if (!t.has_value() || !t->defined()) return nullptr;
  return reinterpret_cast<T*>(t->data_ptr());
}

// x: [rows, K] or [G, cap, K] bf16 -> q [.., K/2] uint8, sf (scale atoms), gscale [rows] fp32
void quant_act_nvfp4(const Tensor& x, const Tensor& q, const Tensor& sf, const Tensor& gscale,
                     const c10::optional<Tensor>& group_counts, const c10::optional<Tensor>& ag_flags,
                     int64_t ag_expected, const c10::optional<Tensor>& ag_ticket, const Tensor& status,
                     int64_t spin_limit) {
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == torch::kBFloat16 && x.stride(-1) == 1, "quant_act_nvfp4: bf16 rows");
  const int64_t K = x.size(-1);
  TORCH_CHECK(K % 64 == 0, "quant_act_nvfp4: K must be a multiple of 64");
  const int64_t G = x.dim() == 3 ? x.size(0) : 1;
  const int64_t R = x.size(-2);
  TORCH_CHECK(x.dim() == 2 || x.stride(0) == R * x.stride(1), "quant_act_nvfp4: groups must be dense");
  TORCH_CHECK(G == 1 || R % 128 == 0, "quant_act_nvfp4: grouped rows must be a multiple of 128 per group");
  const int64_t tiles = (G * R + 127) / 128;
  TORCH_CHECK(q.scalar_type() == torch::kUInt8 && q.is_contiguous() && q.numel() >= G * R * K / 2, "quant_act_nvfp4: q");
  TORCH_CHECK(sf.scalar_type() == torch::kUInt8 && sf.is_contiguous() && sf.numel() >= tiles * (K / 64) * 512,
              "quant_act_nvfp4: sf too small");
  TORCH_CHECK(gscale.scalar_type() == torch::kFloat32 && gscale.numel() >= G * R, "quant_act_nvfp4: gscale");
  oxb::QuantActWait wait{};
  if (ag_flags.has_value() && ag_flags->defined()) {
    TORCH_CHECK(ag_ticket.has_value() && ag_ticket->defined(), "quant_act_nvfp4: ag_ticket required with ag_flags");
    wait.flags = reinterpret_cast<const uint32_t*>(ag_flags->data_ptr());
    wait.n_src = static_cast<int>(ag_flags->numel());
    wait.expected = static_cast<uint32_t>(ag_expected);
    wait.ticket = reinterpret_cast<uint32_t*>(ag_ticket->data_ptr());
    wait.status = reinterpret_cast<int*>(status.data_ptr());
  }
  oxb::launch_quant_act_nvfp4(reinterpret_cast<const __nv_bfloat16*>(x.data_ptr()), x.stride(-2), q.data_ptr<uint8_t>(),
                              sf.data_ptr<uint8_t>(), gscale.data_ptr<float>(), static_cast<int>(G),
                              static_cast<int>(R), static_cast<int>(K), opt_ptr<uint32_t>(group_counts), wait,
                              static_cast<uint32_t>(spin_limit > 0 ? spin_limit : 0), cur_stream());
  check_launch("quant_act_nvfp4");
}

// a8: [M, K] e4m3 bytes; sa_t: [ceil(K/128), >= M] fp32; w8: [N, K] e4m3 bytes; sw: [ceil(N/128), ceil(K/128)].
void gemm_fp8_block(const Tensor& a8, const Tensor& sa_t, const Tensor& w8, const Tensor& sw,
                    const c10::optional<Tensor>& out_opt, const c10::optional<Tensor>& bias,
                    const Tensor& status, const std::vector<int64_t>& slab_ptrs,
                    const std::vector<int64_t>& arrive_ptrs, const c10::optional<Tensor>& done_ticket,
                    int64_t rows_per_owner, int64_t my_rank, int64_t slab_ld) {
  TORCH_CHECK(a8.is_cuda() && w8.is_cuda() && a8.element_size() == 1 && w8.element_size() == 1,
              "gemm_fp8_block: CUDA fp8 operands required");
  TORCH_CHECK(a8.dim() == 2 && w8.dim() == 2 && a8.stride(1) == 1 && w8.stride(1) == 1,
              "gemm_fp8_block: row-major 2-D operands required");
  const int64_t M = a8.size(0), K = a8.size(1), N = w8.size(0);
  TORCH_CHECK(w8.size(1) == K && K % 16 == 0, "gemm_fp8_block: K mismatch or K % 16 != 0");
  const int64_t n_kb = (K + 127) / 128;
  TORCH_CHECK(sa_t.scalar_type() == torch::kFloat32 && sa_t.dim() == 2 && sa_t.size(0) == n_kb &&
                  sa_t.size(1) >= M && sa_t.stride(1) == 1,
              "gemm_fp8_block: sa_t must be [K/128, >=M] fp32");
  TORCH_CHECK(sw.scalar_type() == torch::kFloat32 && sw.is_contiguous() &&
                  sw.size(0) == (N + 127) / 128 && sw.size(1) == n_kb,
              "gemm_fp8_block: sw must be [N/128, K/128] fp32");
  const bool routed = !slab_ptrs.empty();
  if (!routed) {
    TORCH_CHECK(out_opt.has_value(), "gemm_fp8_block: out required");
    const Tensor& out = *out_opt;
    TORCH_CHECK(out.scalar_type() == torch::kBFloat16 && out.size(0) == M && out.size(1) == N &&
                    out.stride(1) == 1,
                "gemm_fp8_block: out must be [M, N] bf16");
  } else {
    TORCH_CHECK(slab_ptrs.size() <= 8 && rows_per_owner > 0 && slab_ld >= N,
                "gemm_fp8_block: 1..8 owners, rows_per_owner > 0, slab_ld >= N");
  }
  CUtensorMap tmA = oxb::make_tma_map(a8.data_ptr(), CU_TENSOR_MAP_DATA_TYPE_UINT8, 1, 2, K, M, 1,
                                      static_cast<uint64_t>(a8.stride(0)), 0, 128, 128, 1,
                                      CU_TENSOR_MAP_SWIZZLE_128B);
  CUtensorMap tmB = oxb::make_tma_map(w8.data_ptr(), CU_TENSOR_MAP_DATA_TYPE_UINT8, 1, 2, K, N, 1,
                                      static_cast<uint64_t>(w8.stride(0)), 0, 128, 128, 1,
                                      CU_TENSOR_MAP_SWIZZLE_128B);
  oxb::Fp8GemmParams p{};
  p.M = static_cast<int>(M);
  p.N = static_cast<int>(N);
  p.K = static_cast<int>(K);
  p.sa_t = sa_t.data_ptr<float>();
  p.sa_ld = static_cast<int>(sa_t.stride(0));
  p.sw = sw.data_ptr<float>();
  if (!routed) {
    p.C = reinterpret_cast<__nv_bfloat16*>(out_opt->data_ptr());
    p.ldc = out_opt->stride(0);
  } else {
    for (size_t i = 0; i < slab_ptrs.size(); ++i) p.slab[i] = reinterpret_cast<__nv_bfloat16*>(slab_ptrs[i]);
    for (size_t i = 0; i < arrive_ptrs.size() && i < 8; ++i)
      p.arrive[i] = reinterpret_cast<uint32_t*>(arrive_ptrs[i]);
    p.n_owners = static_cast<int>(slab_ptrs.size());
    p.rows_per_owner = static_cast<int>(rows_per_owner);
    p.my_rank = static_cast<int>(my_rank);
    p.slab_ld = slab_ld;
    p.done_ticket = opt_ptr<uint32_t>(done_ticket);
  }
  p.bias = bf16_ptr(bias);
  p.status = reinterpret_cast<int*>(status.data_ptr());
  oxb::launch_gemm_fp8_block(tmA, tmB, p, cur_stream());
  check_launch("gemm_fp8_block");
}

void quant_act_fp8(const Tensor& x, const Tensor& q, const Tensor& sa_t,
                   const c10::optional<Tensor>& ag_flags, int64_t ag_expected, int64_t ag_rows_per_src,
                   const c10::optional<Tensor>& ag_ticket, const Tensor& status) {
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == torch::kBFloat16 && x.dim() == 2 && x.stride(1) == 1,
              "quant_act_fp8: [M, K] bf16 input required");
  TORCH_CHECK(q.element_size() == 1 && q.size(0) == x.size(0) && q.size(1) == x.size(1) &&
                  q.stride(1) == 1,
              "quant_act_fp8: q must be [M, K] bytes");
  TORCH_CHECK(sa_t.scalar_type() == torch::kFloat32 && sa_t.size(0) == (x.size(1) + 127) / 128 &&
                  sa_t.size(1) >= x.size(0) && sa_t.stride(1) == 1,
              "quant_act_fp8: sa_t must be [K/128, >=M] fp32");
  oxb::QuantActWait wait{};
  if (ag_flags.has_value() && ag_flags->defined()) {
    TORCH_CHECK(ag_ticket.has_value(), "quant_act_fp8: ag_ticket required with ag_flags");
    wait.flags = reinterpret_cast<const uint32_t*>(ag_flags->data_ptr());
    wait.n_src = static_cast<int>(ag_flags->numel());
    wait.expected = static_cast<uint32_t>(ag_expected);
    wait.rows_per_src = static_cast<int>(ag_rows_per_src);
    wait.ticket = reinterpret_cast<uint32_t*>(ag_ticket->data_ptr());
    wait.status = reinterpret_cast<int*>(status.data_ptr());
  }
  oxb::launch_quant_act_fp8(reinterpret_cast<const __nv_bfloat16*>(x.data_ptr()), x.stride(0),
                            reinterpret_cast<uint8_t*>(q.data_ptr()), q.stride(0),
                            sa_t.data_ptr<float>(), static_cast<int>(sa_t.stride(0)),
                            static_cast<int>(x.size(0)), static_cast<int>(x.size(1)), wait, cur_stream());
  check_launch("quant_act_fp8");
}

void mmvq(int64_t qtype, const Tensor& w, const Tensor& x, const c10::optional<Tensor>& bias,
          const Tensor& out, int64_t N, int64_t K, bool add, const c10::optional<Tensor>& xq,
          const c10::optional<Tensor>& xd, const c10::optional<Tensor>& xs) {
  TORCH_CHECK(w.scalar_type() == torch::kUInt8 && w.is_cuda(), "mmvq: packed uint8 weights");
  TORCH_CHECK(K % 32 == 0, "mmvq: K must be a multiple of 32");
  oxb::MmvqParams p{};
  p.w = w.data_ptr<uint8_t>();
  p.row_bytes = oxb::quant_row_bytes(static_cast<int>(qtype), K);
  TORCH_CHECK(p.row_bytes > 0 && w.numel() >= p.row_bytes * N, "mmvq: weight buffer too small");
  p.x = bf16_ptr(x);
  p.ldx = x.stride(0);
  p.bias = bf16_ptr(bias);
  if (out.scalar_type() == torch::kFloat32)
    p.out_f32 = out.data_ptr<float>();
  else
    p.out_bf16 = reinterpret_cast<__nv_bfloat16*>(out.data_ptr());
  p.ldo = out.stride(0);
  p.M = static_cast<int>(x.size(0));
  p.N = static_cast<int>(N);
  p.K = static_cast<int>(K);
  p.add = add ? 1 : 0;
  if (xq.has_value() && xq->defined()) {
    TORCH_CHECK(xd.has_value() && xs.has_value() && xq->element_size() == 1 && xq->is_contiguous() &&
                    xq->size(0) >= x.size(0) && xq->size(1) == K && xd->is_contiguous() &&
                    xs->is_contiguous() && xd->size(1) == K / 32 && xs->size(1) == K / 32,
                "mmvq: xq [M, K] int8 with xd / xs [M, K/32] fp32 expected");
    p.xq = reinterpret_cast<const int8_t*>(xq->data_ptr());
    p.xd = xd->data_ptr<float>();
    p.xs = xs->data_ptr<float>();
  }
  TORCH_CHECK(oxb::launch_mmvq(static_cast<int>(qtype), p, cur_stream()),
              "mmvq: no device decoder for GGUF type ", qtype);
  check_launch("mmvq");
}

// Stacked packed matrices of different block types sharing K (one launch): out[:, sum of n_i].
void mmvq_mixed(const std::vector<int64_t>& qtypes, const std::vector<Tensor>& ws, const std::vector<int64_t>& ns,
                const Tensor& x, const Tensor& out, int64_t K, const Tensor& xq, const Tensor& xd,
                const Tensor& xs) {
  const size_t n_seg = qtypes.size();
  TORCH_CHECK(n_seg >= 1 && n_seg <= 4 && ws.size() == n_seg && ns.size() == n_seg, "mmvq_mixed: 1..4 segments");
  TORCH_CHECK(K % 32 == 0, "mmvq_mixed: K must be a multiple of 32");
  oxb::MmvqParams p{};
  int64_t rows = 0;
  for (size_t i = 0; i < n_seg; ++i) {
    TORCH_CHECK(ws[i].scalar_type() == torch::kUInt8 && ws[i].is_cuda(), "mmvq_mixed: packed uint8 weights");
    p.seg_type[i] = static_cast<int>(qtypes[i]);
    p.seg_w[i] = ws[i].data_ptr<uint8_t>();
    p.seg_row_bytes[i] = oxb::quant_row_bytes(p.seg_type[i], K);
    TORCH_CHECK(p.seg_row_bytes[i] > 0 && ws[i].numel() >= p.seg_row_bytes[i] * ns[i],
                "mmvq_mixed: weight buffer ", i, " too small");
    rows += ns[i];
    p.seg_row_end[i] = static_cast<int>(rows);
  }
  p.n_seg = static_cast<int>(n_seg);
  p.x = bf16_ptr(x);
  p.ldx = x.stride(0);
  if (out.scalar_type() == torch::kFloat32)
    p.out_f32 = out.data_ptr<float>();
  else
    p.out_bf16 = reinterpret_cast<__nv_bfloat16*>(out.data_ptr());
  TORCH_CHECK(out.size(1) >= rows && out.size(0) >= x.size(0), "mmvq_mixed: out too small");
  p.ldo = out.stride(0);
  p.M = static_cast<int>(x.size(0));
  p.N = static_cast<int>(rows);
  p.K = static_cast<int>(K);
  TORCH_CHECK(xq.element_size() == 1 && xq.is_contiguous() && xq.size(0) >= x.size(0) && xq.size(1) == K &&
                  xd.is_contiguous() && xs.is_contiguous() && xd.size(1) == K / 32 && xs.size(1) == K / 32,
              "mmvq_mixed: xq [M, K] int8 with xd / xs [M, K/32] fp32 expected");
  p.xq = reinterpret_cast<const int8_t*>(xq.data_ptr());
  p.xd = xd.data_ptr<float>();
  p.xs = xs.data_ptr<float>();
  TORCH_CHECK(oxb::launch_mmvq_mixed(p, cur_stream()),
              "mmvq_mixed: a segment's block type has no integer path or an operand is misaligned");
  check_launch("mmvq_mixed");
}

void quant_q8_1(const Tensor& x, const Tensor& xq, const Tensor& xd, const Tensor& xs) {
  TORCH_CHECK(x.is_cuda() && x.scalar_type() == torch::kBFloat16 && x.dim() == 2 && x.stride(1) == 1 &&
                  x.size(1) % 32 == 0,
              "quant_q8_1: [M, K] bf16 input with K % 32 == 0");
  const int64_t M = x.size(0), K = x.size(1);
  TORCH_CHECK(xq.element_size() == 1 && xq.is_contiguous() && xq.size(0) >= M && xq.size(1) == K &&
                  xd.scalar_type() == torch::kFloat32 && xd.is_contiguous() && xd.size(0) >= M &&
                  xd.size(1) == K / 32 && xs.scalar_type() == torch::kFloat32 && xs.is_contiguous() &&
                  xs.size(0) >= M && xs.size(1) == K / 32,
              "quant_q8_1: xq [M, K] int8, xd / xs [M, K/32] fp32");
  oxb::launch_quant_q8_1(reinterpret_cast<const __nv_bfloat16*>(x.data_ptr()), x.stride(0),
                         reinterpret_cast<int8_t*>(xq.data_ptr()), xd.data_ptr<float>(),
                         xs.data_ptr<float>(), static_cast<int>(M), static_cast<int>(K), cur_stream());
  check_launch("quant_q8_1");
}

void dequant_rows(int64_t qtype, const Tensor& w, const c10::optional<Tensor>& row_ids,
                  const Tensor& out, int64_t n_src_rows, int64_t K, double scale) {
  TORCH_CHECK(w.scalar_type() == torch::kUInt8 && w.is_cuda(), "dequant_rows: packed weights");
  TORCH_CHECK(K % 32 == 0, "dequant_rows: K must be a multiple of 32");
  const long long rb = oxb::quant_row_bytes(static_cast<int>(qtype), K);
  const int* ids = nullptr;
  if (row_ids.has_value() && row_ids->defined()) ids = row_ids->data_ptr<int>();
  TORCH_CHECK(oxb::launch_dequant_rows(static_cast<int>(qtype), w.data_ptr<uint8_t>(), rb, ids,
                                       static_cast<int>(out.size(0)), static_cast<int>(K),
                                       reinterpret_cast<__nv_bfloat16*>(out.data_ptr()),
                                       out.stride(0), static_cast<float>(scale),
                                       static_cast<int>(n_src_rows), cur_stream()),
              "dequant_rows: no device decoder for GGUF type ", qtype);
  check_launch("dequant_rows");
}

int64_t quant_row_bytes(int64_t qtype, int64_t K) {
  return oxb::quant_row_bytes(static_cast<int>(qtype), K);
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
  m.doc() = "sm_100a kernels for quantised weights";
  m.def("set_pdl", [](bool on) { oxb::pdl_enabled() = on; });
  m.def("quant_act_nvfp4", &quant_act_nvfp4);
  m.def("gemm_fp8_block", &gemm_fp8_block);
  m.def("quant_act_fp8", &quant_act_fp8);
  m.def("mmvq_mixed", &mmvq_mixed);
  m.def("mmvq", &mmvq);
  m.def("quant_q8_1", &quant_q8_1);
  m.def("dequant_rows", &dequant_rows);
  m.def("quant_row_bytes", &quant_row_bytes);
  m.def("mmvq_has_int8_path", [](int64_t t) { return oxb::mmvq_has_int8_path(static_cast<int>(t)); });
}

// Projection GEMM of the tower: out (rows, out_features) = x (rows, in_features) . w (out_features,
// in_features)^T, one cuBLASLt call.  A library GEMM - the reference's own choice for its projections
// (src/ops/cuda/linear.cu:105-203) and outside the rewritten path; it is here so that the native
// runtime and the torch-tensor mirror share one tuned call: on the first use of a shape up to eight
// heuristic candidates are timed on the real operands and the fastest is kept (at a few dozen rows
// the heuristic's first choice is often not it).
#include <cublasLt.h>
#include <cuda_runtime.h>
#include <dlfcn.h>
#include <stdint.h>

#include <array>
#include <map>
#include <mutex>

#include "axono_b200.h"

namespace {

// cuBLASLt is opened on first use, by its soname first: a process that also holds PyTorch then shares
// the copy PyTorch loaded (two different builds under one soname cannot live side by side - import
// torch before the first projection in such a process), and a process without it gets the toolkit's.
struct LtApi {
  decltype(&cublasLtCreate) Create = nullptr;
  decltype(&cublasLtMatmulDescCreate) DescCreate = nullptr;
  decltype(&cublasLtMatmulDescSetAttribute) DescSet = nullptr;
  decltype(&cublasLtMatrixLayoutCreate) LayoutCreate = nullptr;
  decltype(&cublasLtMatrixLayoutSetAttribute) LayoutSet = nullptr;
  decltype(&cublasLtMatmulPreferenceCreate) PrefCreate = nullptr;
  decltype(&cublasLtMatmulPreferenceSetAttribute) PrefSet = nullptr;
  decltype(&cublasLtMatmulPreferenceDestroy) PrefDestroy = nullptr;
  decltype(&cublasLtMatmulAlgoGetHeuristic) Heuristic = nullptr;
  decltype(&cublasLtMatmul) Matmul = nullptr;
  bool ok = false;
};
const LtApi &lt_api() {
  static LtApi api = [] {
    LtApi a;
    void *h = dlopen("libcublasLt.so.12", RTLD_NOW | RTLD_GLOBAL);
    if (!h) h = dlopen("/usr/local/cuda/lib64/libcublasLt.so.12", RTLD_NOW | RTLD_GLOBAL);
    if (!h) return a;
#define AXONO_LT_SYM(field, name) a.field = reinterpret_cast<decltype(a.field)>(dlsym(h, #name))
    AXONO_LT_SYM(Create, cublasLtCreate);
    AXONO_LT_SYM(DescCreate, cublasLtMatmulDescCreate);
    AXONO_LT_SYM(DescSet, cublasLtMatmulDescSetAttribute);
    AXONO_LT_SYM(LayoutCreate, cublasLtMatrixLayoutCreate);
    AXONO_LT_SYM(LayoutSet, cublasLtMatrixLayoutSetAttribute);
    AXONO_LT_SYM(PrefCreate, cublasLtMatmulPreferenceCreate);
    AXONO_LT_SYM(PrefSet, cublasLtMatmulPreferenceSetAttribute);
    AXONO_LT_SYM(PrefDestroy, cublasLtMatmulPreferenceDestroy);
    AXONO_LT_SYM(Heuristic, cublasLtMatmulAlgoGetHeuristic);
    AXONO_LT_SYM(Matmul, cublasLtMatmul);
#undef AXONO_LT_SYM
    a.ok = a.Create && a.DescCreate && a.DescSet && a.LayoutCreate && a.LayoutSet && a.PrefCreate && a.PrefSet && a.PrefDestroy &&
           a.Heuristic && a.Matmul;
    return a;
  }();
  return api;
}

// One cuBLASLt handle and one 32 MB workspace per device, made on first use (outside graph capture:
// the warm-up run of CUDAGraph.capture makes that first call); one matmul plan per shape, layout, types and
// alignment class.  The workspace is shared by every call on the device: calls that may overlap on the
// GPU (different streams) would race on it - keep the projections of one device on one stream.
struct LtState {
  cublasLtHandle_t handle = nullptr;
  void *workspace = nullptr;
  size_t workspace_bytes = size_t(32) << 20;
  struct Plan {
    cublasLtMatmulDesc_t op = nullptr;
    cublasLtMatrixLayout_t a = nullptr, b = nullptr, c = nullptr;
    cublasLtMatmulAlgo_t algo;
  };
  std::map<std::array<int64_t, 12>, Plan> plans;
};
std::mutex g_lt_mu;
LtState g_lt[64];


// `batch` products out[b] (rows, outf) = x[b] (rows, in) . w[b]^T of row-major operands with row strides and
// batch strides in elements; w[b] is stored (outf, in), or (in, outf) with w_in_major.
struct Gemm {
  int64_t rows, outf, in, x_ld, w_ld, out_ld, batch, x_stride, w_stride, out_stride;
  bool w_in_major;
  int dtype, out_dtype;
  bool timed;  // time the heuristic's candidates on first use (else its first choice)
};

cudaDataType_t lt_type(int dtype) {
  return dtype == AXB200_FLOAT16 ? CUDA_R_16F : dtype == AXB200_BFLOAT16 ? CUDA_R_16BF : CUDA_R_32F;
}
bool lt_known(int dtype) { return dtype == AXB200_FLOAT16 || dtype == AXB200_BFLOAT16 || dtype == AXB200_FLOAT32; }

int run_gemm(const Gemm &g, const void *x, const void *w, void *out, void *stream) {
  if (!x || !w || !out) return AXB200_INVALID_PTR;
  if (g.rows <= 0 || g.outf <= 0 || g.in <= 0 || g.batch <= 0) return AXB200_INVALID_ARGUMENT;
  if (g.x_ld < g.in || g.out_ld < g.outf || g.w_ld < (g.w_in_major ? g.outf : g.in)) return AXB200_SHAPE_MISMATCH;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  cudaStreamCaptureStatus cap = cudaStreamCaptureStatusNone;
  if (cudaStreamIsCapturing(st, &cap) != cudaSuccess) return AXB200_DEVICE_ERROR;
  const bool capturing = cap != cudaStreamCaptureStatusNone;
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return AXB200_DEVICE_ERROR;
  const LtApi &api = lt_api();
  if (!api.ok) return AXB200_INTERNAL_ERROR;
  std::lock_guard<std::mutex> lock(g_lt_mu);
  LtState &lt = g_lt[dev];
  if (!lt.handle) {
    if (capturing) return AXB200_INVALID_ARGUMENT;  // first use must be outside a capture
    // the workspace first: a handle is only published together with the memory every later call assumes
    void *ws = nullptr;
    if (cudaMalloc(&ws, lt.workspace_bytes) != cudaSuccess) {
      cudaGetLastError();
      return AXB200_OUT_OF_MEMORY;
    }
    cublasLtHandle_t h = nullptr;
    if (api.Create(&h) != CUBLAS_STATUS_SUCCESS) {
      cudaFree(ws);
      return AXB200_DEVICE_ERROR;
    }
    lt.workspace = ws;
    lt.handle = h;
  }
  const cudaDataType_t dt = lt_type(g.dtype), dt_out = lt_type(g.out_dtype);
  // The algorithm is chosen for the operands' alignment too: a plan made for 256-byte aligned pointers
  // may not be valid for less aligned ones, so the largest power of two (up to 256) that divides all
  // three addresses is part of the plan's key and told to the heuristic.
  const uintptr_t bits = reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out) | 256u;
  const uint32_t align = (uint32_t)(bits & (~bits + 1));
  const std::array<int64_t, 12> key = {g.rows, g.outf, g.in, g.x_ld, g.w_ld, g.out_ld, g.batch, g.x_stride, g.w_stride,
                                       g.out_stride, (int64_t)g.w_in_major, (int64_t)(g.dtype * 16 + g.out_dtype) * 512 + align};
  auto it = lt.plans.find(key);
  if (it == lt.plans.end()) {
    if (capturing) return AXB200_INVALID_ARGUMENT;  // plans are made (and timed) in a warm-up run
    // Row-major result (rows, out) = x . w^T is column-major (out, rows) = w_cm^T . x_cm, where the
    // row-major buffers read column-major are w_cm (in, out) and x_cm (in, rows); a w stored (in, out) is
    // read column-major as (out, in) and taken as it is.
    LtState::Plan pl;
    const cublasOperation_t ta = g.w_in_major ? CUBLAS_OP_N : CUBLAS_OP_T, tb = CUBLAS_OP_N;
    bool ok = api.DescCreate(&pl.op, CUBLAS_COMPUTE_32F, CUDA_R_32F) == CUBLAS_STATUS_SUCCESS;
    ok = ok && api.DescSet(pl.op, CUBLASLT_MATMUL_DESC_TRANSA, &ta, sizeof(ta)) == CUBLAS_STATUS_SUCCESS;
    ok = ok && api.DescSet(pl.op, CUBLASLT_MATMUL_DESC_TRANSB, &tb, sizeof(tb)) == CUBLAS_STATUS_SUCCESS;
    ok = ok && (g.w_in_major ? api.LayoutCreate(&pl.a, dt, g.outf, g.in, g.w_ld)
                             : api.LayoutCreate(&pl.a, dt, g.in, g.outf, g.w_ld)) == CUBLAS_STATUS_SUCCESS;  // w_cm
    ok = ok && api.LayoutCreate(&pl.b, dt, g.in, g.rows, g.x_ld) == CUBLAS_STATUS_SUCCESS;          // x_cm
    ok = ok && api.LayoutCreate(&pl.c, dt_out, g.outf, g.rows, g.out_ld) == CUBLAS_STATUS_SUCCESS;  // result_cm
    if (g.batch > 1) {
      const int32_t count = (int32_t)g.batch;
      const cublasLtMatrixLayout_t lay[3] = {pl.a, pl.b, pl.c};
      const int64_t stride[3] = {g.w_stride, g.x_stride, g.out_stride};
      for (int i = 0; i < 3 && ok; ++i)
        ok = api.LayoutSet(lay[i], CUBLASLT_MATRIX_LAYOUT_BATCH_COUNT, &count, sizeof(count)) == CUBLAS_STATUS_SUCCESS &&
             api.LayoutSet(lay[i], CUBLASLT_MATRIX_LAYOUT_STRIDED_BATCH_OFFSET, &stride[i], sizeof(stride[i])) ==
                 CUBLAS_STATUS_SUCCESS;
    }
    cublasLtMatmulPreference_t pref = nullptr;
    ok = ok && api.PrefCreate(&pref) == CUBLAS_STATUS_SUCCESS;
    ok = ok && api.PrefSet(pref, CUBLASLT_MATMUL_PREF_MAX_WORKSPACE_BYTES, &lt.workspace_bytes,
                                                    sizeof(lt.workspace_bytes)) == CUBLAS_STATUS_SUCCESS;
    for (const auto attr : {CUBLASLT_MATMUL_PREF_MIN_ALIGNMENT_A_BYTES, CUBLASLT_MATMUL_PREF_MIN_ALIGNMENT_B_BYTES,
                            CUBLASLT_MATMUL_PREF_MIN_ALIGNMENT_C_BYTES, CUBLASLT_MATMUL_PREF_MIN_ALIGNMENT_D_BYTES})
      ok = ok && api.PrefSet(pref, attr, &align, sizeof(align)) == CUBLAS_STATUS_SUCCESS;
    // Up to eight candidates from the heuristic, each timed on the real operands (beta = 0, so the
    // trial runs are idempotent): at a few dozen rows the first candidate is often not the fastest.
    constexpr int kCandidates = 8;
    cublasLtMatmulHeuristicResult_t heur[kCandidates];
    int found = 0;
    ok = ok && api.Heuristic(lt.handle, pl.op, pl.a, pl.b, pl.c, pl.c, pref, kCandidates, heur, &found) ==
                   CUBLAS_STATUS_SUCCESS && found > 0;
    if (pref) api.PrefDestroy(pref);
    if (!ok) return AXB200_INTERNAL_ERROR;
    int best = -1;
    for (int c = 0; c < found && best < 0; ++c)  // the first usable candidate, unless a timed one beats it
      if (heur[c].state == CUBLAS_STATUS_SUCCESS && heur[c].workspaceSize <= lt.workspace_bytes) best = c;
    if (best < 0) return AXB200_INTERNAL_ERROR;  // nothing the library offers fits
    if (found > 1 && g.timed) {
      const float one = 1.f, zero = 0.f;
      cudaStream_t ts = st;
      cudaEvent_t e0 = nullptr, e1 = nullptr;
      float best_ms = -1.f;
      if (cudaEventCreate(&e0) == cudaSuccess && cudaEventCreate(&e1) == cudaSuccess) {
        for (int c = 0; c < found; ++c) {
          if (heur[c].state != CUBLAS_STATUS_SUCCESS || heur[c].workspaceSize > lt.workspace_bytes) continue;
          bool run_ok = true;
          for (int rep = 0; rep < 13 && run_ok; ++rep) {
            if (rep == 3) cudaEventRecord(e0, ts);  // three warm-up runs, ten timed
            run_ok = api.Matmul(lt.handle, pl.op, &one, w, pl.a, x, pl.b, &zero, out, pl.c,
                                out, pl.c, &heur[c].algo, lt.workspace, lt.workspace_bytes, ts) ==
                     CUBLAS_STATUS_SUCCESS;
          }
          float ms = 0.f;
          if (!run_ok || cudaEventRecord(e1, ts) != cudaSuccess || cudaEventSynchronize(e1) != cudaSuccess ||
              cudaEventElapsedTime(&ms, e0, e1) != cudaSuccess) {
            cudaGetLastError();
            continue;
          }
          if (best_ms < 0.f || ms < best_ms) {
            best_ms = ms;
            best = c;
          }
        }
      }
      if (e0) cudaEventDestroy(e0);
      if (e1) cudaEventDestroy(e1);
    }
    pl.algo = heur[best].algo;
    it = lt.plans.emplace(key, pl).first;
  }
  const LtState::Plan &pl = it->second;
  const float alpha = 1.f, beta = 0.f;
  const cublasStatus_t cs = api.Matmul(lt.handle, pl.op, &alpha, w, pl.a, x, pl.b, &beta, out, pl.c, out, pl.c, &pl.algo,
                                       lt.workspace, lt.workspace_bytes, st);
  return cs == CUBLAS_STATUS_SUCCESS ? AXB200_OK : AXB200_DEVICE_ERROR;
}

}  // namespace

extern "C" int axb200_linear_nobias(const void *x, const void *w, void *out, int64_t rows, int64_t out_features,
                                    int64_t in_features, int dtype, void *stream) {
  if (!lt_known(dtype)) return AXB200_UNSUPPORTED_TYPE;
  return run_gemm({rows, out_features, in_features, in_features, in_features, out_features, 1, 0, 0, 0, false, dtype, dtype, true},
                  x, w, out, stream);
}

extern "C" int axb200_linear_strided(const void *x, const void *w, void *out, int64_t rows, int64_t out_features,
                                     int64_t in_features, int64_t x_ld, int64_t w_ld, int64_t out_ld, int64_t batch,
                                     int64_t x_stride, int64_t w_stride, int64_t out_stride, int w_in_major, int dtype,
                                     int out_dtype, void *stream) {
  if (!lt_known(dtype) || (out_dtype != dtype && out_dtype != AXB200_FLOAT32)) return AXB200_UNSUPPORTED_TYPE;
  return run_gemm({rows, out_features, in_features, x_ld, w_ld, out_ld, batch, x_stride, w_stride, out_stride, w_in_major != 0,
                   dtype, out_dtype, rows <= 512},
                  x, w, out, stream);
}

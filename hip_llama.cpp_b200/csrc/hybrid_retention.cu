// Retention (tha_retention_t): S_t = decay S_(t-1) + k_t v_t^T with one fixed decay per head, o_t = S_t^T q_t.
//   hyb_rotate_qk_kernel   q and k columns of the stacked projection rotated in place, k scaled by dim^(-1/2)
//   the recurrence         hybrid_gla.cu, SCAN_HEAD_DECAY
// The head norm (no weight) and the silu gate follow in tha_hyb_head_gate.
#include <cuda_bf16.h>

#include "common.cuh"
#include "hybrid_ops.cuh"
#include "tha_hybrid.h"

namespace tha {

// a block per row; work item = one pair of rotated channels, or one channel that passes unchanged, of one head of q or k
__global__ void hyb_rotate_qk_kernel(float* __restrict__ proj, long long ldp, int o_q, int o_k, int heads, int dim, int rot_dims, int layout,
                                     const float* __restrict__ cos_t, const float* __restrict__ sin_t, float k_scale) {
  const int r = blockIdx.x, half = rot_dims >> 1, per = half + (dim - rot_dims);
  float* row = proj + (size_t)r * ldp;
  const float* c = cos_t + (size_t)r * half;
  const float* s = sin_t + (size_t)r * half;
  for (int i = threadIdx.x; i < 2 * heads * per; i += blockDim.x) {
    const bool is_k = i >= heads * per;
    const int j = is_k ? i - heads * per : i;
    const int h = j / per, e = j - h * per;
    const float f = is_k ? k_scale : 1.0f;
    float* p = row + (is_k ? o_k : o_q) + h * dim;
    if (e < half) {
      const int a = layout == THA_ROT_HALVES ? e : 2 * e, b = layout == THA_ROT_HALVES ? e + half : 2 * e + 1;
      const float x = p[a], y = p[b];
      p[a] = (x * c[e] - y * s[e]) * f;
      p[b] = (y * c[e] + x * s[e]) * f;
    } else if (is_k) {
      p[rot_dims + e - half] *= f;
    }
  }
}

}  // namespace tha

using namespace tha;

extern "C" int tha_hyb_retention_scan(void* stream, int dtype, const tha_retention_t* g, const tha_rows_t* rows, const tha_state_store_t* st,
                                      float* proj, long long ldp, const float* cos_t, const float* sin_t, int rot_dims, float* o_raw, void* out, float* seg_scratch, size_t seg_scratch_floats) {
  if (rows->n_seqs < 1 || rows->n_rows < 1) return THA_STATUS_SUCCESS;
  if (g->heads < 1 || g->dim < 1 || g->vdim < 1 || rot_dims > g->dim || (rot_dims & 1)) return THA_STATUS_INVALID_ARG;
  if (g->dim > 512) return THA_STATUS_NOT_SUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
  THA_CUDA_OK(launch(hyb_rotate_qk_kernel, dim3(rows->n_rows), dim3(256), 0, s, false, proj, ldp, g->o_q, g->o_k, g->heads, g->dim, rot_dims,
                     g->rot_layout, cos_t, sin_t, 1.0f / sqrtf((float)g->dim)));
  tha_gla_t a = {};
  a.heads = g->heads; a.dim = g->dim; a.vdim = g->vdim; a.o_q = g->o_q; a.o_k = g->o_k; a.o_v = g->o_v; a.state_off = g->state_off;
  const int status = hyb_scan_launch(s, SCAN_HEAD_DECAY, &a, rows, st, proj, ldp, nullptr, g->decay, o_raw, 1.0f, seg_scratch, seg_scratch_floats);
  if (status != THA_STATUS_SUCCESS) return status;
  return tha_hyb_head_gate(stream, dtype, out, o_raw, rows->n_rows, g->heads, g->vdim, 1, g->eps, nullptr, 0, proj + g->o_g, ldp, THA_GATE_SILU);
}

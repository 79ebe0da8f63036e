// Token-shifted key-value memory (tha_wkv_t).
//   hyb_token_shift_kernel   every row's mixes with its predecessor, h + (h' - h) * mu, n of them in one pass: the inputs of the grouped
//                            product (tha_hyb_linear_groups).  The predecessor of a portion's first row is the slot's stored row.
//   hyb_wkv_decay_kernel     the low-rank decay from end to end: tanh of the W_w1 columns on the way into shared memory, the product with
//                            W_w2 (fp32 FMA, k ascending), and exp(-exp(. + w0)) on the way out
//   the recurrence           hybrid_gla.cu, SCAN_BONUS
// Mixes are formed from the fp32 norm and rounded once, to the product's number format; decays, state and read-out are fp32 in both
// number formats.  The head norm, its weight and the silu gate follow in tha_hyb_head_gate.
#include <cuda_bf16.h>

#include "common.cuh"
#include "hybrid_ops.cuh"
#include "tha_hybrid.h"

namespace tha {

template <int V, typename T>
__device__ __forceinline__ void shift_store(T* p, const float* v) {
  if (V == 4 && sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else if (V == 4) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
  } else {
    hyb_store(p, v[0]);
  }
}
template <int V>
__device__ __forceinline__ void shift_load(const float* p, float* v) {
  if (V == 4) { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
  else v[0] = *p;
}

template <typename T, int V>
__global__ void hyb_token_shift_kernel(tha_rows_t rows, tha_state_store_t st, long long state_off, const float* __restrict__ h, int width,
                                       const float* __restrict__ mu, int n_mix, T* __restrict__ out) {
  const int c = V * (blockIdx.y * blockDim.x + threadIdx.x), r = blockIdx.x;
  if (c >= width) return;
  const int s = rows.row_seq[r];
  const bool inside = r > rows.seq_first[s];
  const float* before = inside ? h + (size_t)(r - 1) * width + c : st.base + (size_t)rows.seq_slot[s] * st.slot_floats + state_off + c;
  float cur[V], d[V], m[V], y[V];
  shift_load<V>(h + (size_t)r * width + c, cur);
  if (inside) shift_load<V>(before, d);
  else
#pragma unroll
    for (int v = 0; v < V; v++) d[v] = before[v];   // the slot's row need not be 16-byte aligned
#pragma unroll
  for (int v = 0; v < V; v++) d[v] -= cur[v];
  for (int i = 0; i < n_mix; i++) {
    shift_load<V>(mu + (size_t)i * width + c, m);
#pragma unroll
    for (int v = 0; v < V; v++) y[v] = fmaf(d[v], m[v], cur[v]);
    shift_store<V>(out + ((size_t)i * rows.n_rows + r) * width + c, y);
  }
}

constexpr int WD_T = 64, WD_K = 16;
// decay[r, c] = exp(-exp(sum_k W2[c, k] tanh(z[r, k]) + w0[c])): 64 x 64 tile, 4 x 4 per thread
template <typename T>
__global__ void __launch_bounds__(256) hyb_wkv_decay_kernel(float* __restrict__ decay, const float* __restrict__ z, long long ldz, int rank,
                                                            const T* __restrict__ w2, const float* __restrict__ w0, int n_rows, int n_ch) {
  __shared__ float As[WD_K][WD_T + 4];
  __shared__ float Ws[WD_K][WD_T + 4];
  const int c0 = blockIdx.x * WD_T, r0 = blockIdx.y * WD_T;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < rank; k0 += WD_K) {
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int k = k0 + lk + e;
      As[lk + e][lr] = (r0 + lr < n_rows && k < rank) ? tanhf(z[(size_t)(r0 + lr) * ldz + k]) : 0.f;
      Ws[lk + e][lr] = (c0 + lr < n_ch && k < rank) ? hyb_load(w2 + (size_t)(c0 + lr) * rank + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < WD_K; k++) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; i++) { a[i] = As[k][ty * 4 + i]; b[i] = Ws[k][tx + 16 * i]; }
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int r = r0 + ty * 4 + i;
    if (r >= n_rows) continue;
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int c = c0 + tx + 16 * j;
      if (c < n_ch) decay[(size_t)r * n_ch + c] = expf(-expf(acc[i][j] + w0[c]));
    }
  }
}

}  // namespace tha

using namespace tha;
typedef __nv_bfloat16 bf16;

extern "C" int tha_hyb_token_shift(void* stream, int dtype, const tha_rows_t* rows, const tha_state_store_t* st, long long shift_state_off,
                                   const float* h, int width, const float* mu, int n_mix, void* out) {
  if (rows->n_rows < 1 || n_mix < 1) return THA_STATUS_SUCCESS;
  if (!h || !mu || !out || width < 1) return THA_STATUS_INVALID_ARG;
  cudaStream_t s = (cudaStream_t)stream;
  const bool vec = width % 4 == 0 && aligned16(h) && aligned16(mu) && aligned16(out);
  const dim3 grid(rows->n_rows, ceil_div(vec ? width / 4 : width, 128));
#define SHIFT_GO(T, V) THA_CUDA_OK(launch(hyb_token_shift_kernel<T, V>, grid, dim3(128), 0, s, false, *rows, *st, shift_state_off, h, width, mu, n_mix, (T*)out))
  if (dtype == THA_DT_BF16) { if (vec) SHIFT_GO(bf16, 4); else SHIFT_GO(bf16, 1); }
  else { if (vec) SHIFT_GO(float, 4); else SHIFT_GO(float, 1); }
#undef SHIFT_GO
  return tha_hyb_conv_tail(stream, rows, st, shift_state_off, h, width, 0, width, 2, nullptr);   // a one-row tail
}

extern "C" int tha_hyb_wkv_scan(void* stream, int dtype, const tha_wkv_t* g, const tha_rows_t* rows, const tha_state_store_t* st,
                                const float* proj, long long ldp, float* decay, float* o_raw, void* out, float* seg_scratch, size_t seg_scratch_floats) {
  if (rows->n_seqs < 1 || rows->n_rows < 1) return THA_STATUS_SUCCESS;
  if (g->heads < 1 || g->dim < 1 || g->rank < 1) return THA_STATUS_INVALID_ARG;
  if (g->dim > 512) return THA_STATUS_NOT_SUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
  const int R = rows->n_rows, HD = g->heads * g->dim;
  const dim3 grid(ceil_div(HD, WD_T), ceil_div(R, WD_T));
  if (dtype == THA_DT_BF16)
    THA_CUDA_OK(launch(hyb_wkv_decay_kernel<bf16>, grid, dim3(256), 0, s, false, decay, proj + g->o_w1, ldp, g->rank, (const bf16*)g->w_w2, g->w0, R, HD));
  else
    THA_CUDA_OK(launch(hyb_wkv_decay_kernel<float>, grid, dim3(256), 0, s, false, decay, proj + g->o_w1, ldp, g->rank, (const float*)g->w_w2, g->w0, R, HD));
  tha_gla_t a = {};
  a.heads = g->heads; a.dim = g->dim; a.vdim = g->dim; a.o_q = g->o_r; a.o_k = g->o_k; a.o_v = g->o_v; a.state_off = g->state_off;
  const int status = hyb_scan_launch(s, SCAN_BONUS, &a, rows, st, proj, ldp, decay, g->u, o_raw, 1.0f, seg_scratch, seg_scratch_floats);
  if (status != THA_STATUS_SUCCESS) return status;
  return tha_hyb_head_gate(stream, dtype, out, o_raw, R, g->heads, g->dim, 1, g->eps, g->norm, 1, proj + g->o_g, ldp, THA_GATE_SILU);
}

// Gated linear attention (tha_gla_t): per head S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t / sqrt(dim).
//   hyb_gla_decay_kernel   all rows at once, in place: z + b -> a = sigmoid(z + b)^(1/tau) = exp(-softplus(-(z + b)) / tau)
//   hyb_gla_scan_kernel    the recurrence with the state in registers: a warp owns GLA_COLS value columns of one
//                          (sequence, head), lane l the key channels l, l + 32, ...; the column sums S^T q are warp
//                          shuffles, a token's inputs are fetched several tokens ahead into a ring of registers; no barrier.
//                          The state of a head lies in the slot as [column pair][key channel][2] (a warp's share is one
//                          contiguous run).  It is read from the sequence's slot before its first row of the step and written back
//                          after its last, so a prompt cut anywhere continues exactly where it stopped.
//   hyb_scan_combine_kernel  long portions run as segments side by side: see ScanSegs
// The scan has three forms (SCAN_*): a decay per key channel from an array (gated linear attention, the bounded-forget-gate
// recurrence), one fixed decay per head (retention), and a decay per key channel with a bonus for the current token whose read-out
// sees the state before the token (the token-shifted key-value memory): o = (S + diag(u) k v^T)^T q, then S = diag(a) S + k v^T.
// Decays, state and read-out are fp32 in both number formats; the head norm and the silu gate follow in
// tha_hyb_head_gate.
#include <cuda_bf16.h>
#include <stdlib.h>

#include "common.cuh"
#include "hybrid_ops.cuh"
#include "tha_hybrid.h"

namespace tha {

constexpr int GLA_WARPS = 4, GLA_STATE_PAD = 8;   // a head's value columns are padded to a multiple of 8 in the slot

__global__ void hyb_gla_decay_kernel(float* __restrict__ z, size_t n, int hd, const float* __restrict__ bias, float inv_tau) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float v = z[i] + (bias ? bias[i % hd] : 0.f);
  z[i] = expf(-hyb_softplus(-v) * inv_tau);
}

__global__ void hyb_hgrn_gates_kernel(float* __restrict__ proj, long long ldp, float* __restrict__ decay, size_t n, int hd, int o_q, int o_f,
                                      const float* __restrict__ f_b, const float* __restrict__ lower) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const size_t r = i / hd;
  const int c = (int)(i - r * hd);
  float* row = proj + r * ldp;
  const float q = row[o_q + c];
  row[o_q + c] = q * hyb_sigmoid(q);
  const float z = row[o_f + c] + f_b[c], lo = lower[c];
  const float open = (1.0f - lo) * hyb_sigmoid(-z);   // 1 - f
  decay[i] = 1.0f - open;
  row[o_f + c] = open;
}

// A long portion is cut into segments that run side by side (ScanSegs::len > 0), which the recurrence allows because a segment's end
// state is linear in its start state, S_end = diag(product of its decays) S_start + (its end state from zero):
//   1. LOCAL: every segment but a portion's last leaves its end state from zero (the first one: its true end state) and its decay
//      products in scratch; the first one also leaves a copy of the slot's state in the last one's place there
//   2. hyb_scan_combine_kernel turns the end states into true ones, in order
//   3. every segment runs again from its true start state and writes its read-outs; the last one writes the slot
struct ScanSegs { int len; float* states; float* prods; };   // states [segment][heads][D * EP], prods [segment][heads * D]

// where block x works: sequence s, segment `seg` of its `n_seg`, which rows, and the first scratch entry of the sequence
struct ScanPlace { int s, seg, n_seg, r_begin, r_end, entry; };
__device__ __forceinline__ ScanPlace scan_place(const tha_rows_t& rows, int len, int tile) {
  ScanPlace p;
  p.seg = 0; p.n_seg = 1; p.entry = 0;
  if (len <= 0) {
    p.s = tile; p.r_begin = rows.seq_first[tile]; p.r_end = rows.seq_first[tile + 1];
    return p;
  }
  for (p.s = 0; p.s < rows.n_seqs; p.s++) {
    const int lo = rows.seq_first[p.s], hi = rows.seq_first[p.s + 1];
    p.n_seg = hi - lo > len ? (hi - lo + len - 1) / len : 1;
    if (tile < p.n_seg) {
      p.seg = tile; p.r_begin = lo + tile * len; p.r_end = min(hi, p.r_begin + len);
      return p;
    }
    tile -= p.n_seg;
    if (p.n_seg > 1) p.entry += p.n_seg;
  }
  p.s = -1;
  return p;
}

// VEC consecutive floats (one 32-, 64- or 128-bit load; the caller checks the alignment)
template <int VEC> __device__ __forceinline__ void scan_ld(const float* p, float* o) {
  if (VEC == 4) { const float4 t = *reinterpret_cast<const float4*>(p); o[0] = t.x; o[1] = t.y; o[2] = t.z; o[3] = t.w; }
  else if (VEC == 2) { const float2 t = *reinterpret_cast<const float2*>(p); o[0] = t.x; o[1] = t.y; }
  else o[0] = *p;
}

// VEC: consecutive key channels per lane (lane l owns l * VEC .. of every run of 32 * VEC; VEC > 1 needs dim, offsets and row pitches
// that are multiples of it, and of four value columns), so that a lane's inputs are few wide loads
template <int RPL, int AHEAD, int GLA_COLS, int FORM, bool LOCAL, int VEC>
__global__ void __launch_bounds__(32 * GLA_WARPS) hyb_gla_scan_kernel(tha_gla_t g, tha_rows_t rows, tha_state_store_t st,
                                                                      const float* __restrict__ proj, long long ldp,
                                                                      const float* __restrict__ decay, const float* __restrict__ aux,
                                                                      float* __restrict__ o_raw, float qscale, ScanSegs segs) {
  const int h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int D = g.dim, E = g.vdim;
  const int e0 = (blockIdx.z * GLA_WARPS + warp) * GLA_COLS;
  if (e0 >= E) return;
  const ScanPlace at = scan_place(rows, segs.len, blockIdx.x);
  if (at.s < 0 || (LOCAL && at.seg == at.n_seg - 1)) return;
  // a head's state as [column pair][key channel][2]: a warp's share is one contiguous run
  const int EP = (E + GLA_STATE_PAD - 1) / GLA_STATE_PAD * GLA_STATE_PAD;
  const size_t mine = (size_t)h * D * EP + (size_t)e0 * D, entry = (size_t)g.heads * D * EP;
  float* slot = st.base + (size_t)rows.seq_slot[at.s] * st.slot_floats + g.state_off + mine;
  const float* start = at.n_seg == 1 || (LOCAL && at.seg == 0) ? slot
                       : segs.states + (size_t)(at.entry + (at.seg == 0 ? at.n_seg - 1 : at.seg - 1)) * entry + mine;
  const bool from_zero = LOCAL && at.seg > 0;
  const bool pairs = ((reinterpret_cast<size_t>(slot) | reinterpret_cast<size_t>(segs.states)) & 7) == 0;
  auto ch = [&](int i) { return (i / VEC) * (32 * VEC) + lane * VEC + i % VEC; };   // this lane's i-th key channel
  // a column pair of a channel is one 64-bit word where the regions start on even floats (the loader's do); one branch outside, so
  // that all of a lane's loads are in flight together
  float S[RPL][GLA_COLS];
  if (pairs) {
    float2 t[RPL][GLA_COLS / 2];
#pragma unroll
    for (int i = 0; i < RPL; i++)
#pragma unroll
      for (int c = 0; c < GLA_COLS; c += 2) {
        const bool live = ch(i) < D && e0 + c < E && !from_zero;
        t[i][c / 2] = live ? *reinterpret_cast<const float2*>(start + (size_t)c * D + 2 * ch(i)) : make_float2(0.f, 0.f);
      }
#pragma unroll
    for (int i = 0; i < RPL; i++)
#pragma unroll
      for (int c = 0; c < GLA_COLS; c += 2) { S[i][c] = t[i][c / 2].x; S[i][c + 1] = e0 + c + 1 < E ? t[i][c / 2].y : 0.f; }
  } else {
#pragma unroll
    for (int i = 0; i < RPL; i++)
#pragma unroll
      for (int c = 0; c < GLA_COLS; c++)
        S[i][c] = (ch(i) < D && e0 + c < E && !from_zero) ? start[(size_t)(c >> 1) * 2 * D + 2 * ch(i) + (c & 1)] : 0.f;
  }
  auto leave = [&](float* dst) {
    if (pairs) {
#pragma unroll
      for (int i = 0; i < RPL; i++)
#pragma unroll
        for (int c = 0; c < GLA_COLS; c += 2)   // an odd last column's partner is padding
          if (ch(i) < D && e0 + c < E) *reinterpret_cast<float2*>(dst + (size_t)c * D + 2 * ch(i)) = make_float2(S[i][c], S[i][c + 1]);
    } else {
#pragma unroll
      for (int i = 0; i < RPL; i++)
#pragma unroll
        for (int c = 0; c < GLA_COLS; c++)
          if (ch(i) < D && e0 + c < E) dst[(size_t)(c >> 1) * 2 * D + 2 * ch(i) + (c & 1)] = S[i][c];
    }
  };
  if (LOCAL && at.seg == 0) leave(segs.states + (size_t)(at.entry + at.n_seg - 1) * entry + mine);
  constexpr bool BONUS = FORM == SCAN_BONUS && !LOCAL;
  float fixed_decay = 0.f, bonus[BONUS ? RPL : 1], prod[LOCAL ? RPL : 1];
  if (FORM == SCAN_HEAD_DECAY) fixed_decay = aux[h];
  if (BONUS) {
#pragma unroll
    for (int i = 0; i < RPL; i++) bonus[i] = ch(i) < D ? aux[h * D + ch(i)] : 0.f;
  }
  if (LOCAL) {
#pragma unroll
    for (int i = 0; i < RPL; i++) prod[i] = 1.f;
  }
  const int r_begin = at.r_begin, r_end = at.r_end;
  // a token's inputs are loaded AHEAD tokens before they are used (a ring of register sets, the loop unrolled over it)
  struct In { float q[LOCAL ? 1 : RPL], k[RPL], a[FORM == SCAN_HEAD_DECAY ? 1 : RPL], v[GLA_COLS]; };
  In ring[AHEAD];
  auto fetch = [&](int r, In& in) {
    const float* x = proj + (size_t)r * ldp;
#pragma unroll
    for (int i = 0; i < RPL; i += VEC) {
      const int d = ch(i);
      if (d < D) {
        if (!LOCAL) scan_ld<VEC>(x + g.o_q + h * D + d, in.q + i);
        scan_ld<VEC>(x + g.o_k + h * D + d, in.k + i);
        if (FORM != SCAN_HEAD_DECAY) scan_ld<VEC>(decay + (size_t)r * g.heads * D + h * D + d, in.a + i);
      } else {
#pragma unroll
        for (int v = i; v < i + VEC; v++) {
          if (!LOCAL) in.q[v] = 0.f;
          in.k[v] = 0.f;
          if (FORM != SCAN_HEAD_DECAY) in.a[v] = 0.f;
        }
      }
    }
    if (VEC > 1) {
#pragma unroll
      for (int c = 0; c < GLA_COLS; c += 4) {
        if (e0 + c < E) scan_ld<4>(x + g.o_v + h * E + e0 + c, in.v + c);
        else
#pragma unroll
          for (int v = 0; v < 4; v++) in.v[c + v] = 0.f;
      }
    } else {
#pragma unroll
      for (int c = 0; c < GLA_COLS; c++) in.v[c] = e0 + c < E ? x[g.o_v + h * E + e0 + c] : 0.f;
    }
  };
#pragma unroll
  for (int u = 0; u < AHEAD; u++)
    if (r_begin + u < r_end) fetch(r_begin + u, ring[u]);
  // one token; `refill` (a row, or -1) is what the token's ring entry is loaded with once its values are taken
  auto token = [&](int r, In& in, int refill) {
    float cq[LOCAL ? 1 : RPL], ck[RPL], ca[RPL], cv[GLA_COLS], o[GLA_COLS];
#pragma unroll
    for (int i = 0; i < RPL; i++) {
      if (!LOCAL) cq[i] = in.q[i] * qscale;
      ck[i] = in.k[i];
      ca[i] = FORM == SCAN_HEAD_DECAY ? fixed_decay : in.a[i];
    }
#pragma unroll
    for (int c = 0; c < GLA_COLS; c++) { cv[c] = in.v[c]; o[c] = 0.f; }
    if (refill >= 0) fetch(refill, in);
    if (LOCAL) {
#pragma unroll
      for (int i = 0; i < RPL; i++) prod[i] *= ca[i];
    }
#pragma unroll
    for (int i = 0; i < RPL; i++)
#pragma unroll
      for (int c = 0; c < GLA_COLS; c++) {
        const float kv = ck[i] * cv[c];
        if (BONUS) o[c] = fmaf(fmaf(bonus[i], kv, S[i][c]), cq[i], o[c]);
        S[i][c] = fmaf(S[i][c], ca[i], kv);
        if (!BONUS && !LOCAL) o[c] = fmaf(S[i][c], cq[i], o[c]);
      }
    if (LOCAL) return;
    // the column sums: halve the columns a lane carries while exchanging across lane bits 4, 3, 2 (a lane ends with ONE
    // column, col = its bits [4 : 4 - log2(COLS)]), then finish over the remaining lane bits
    int width = GLA_COLS;
#pragma unroll
    for (int off = 16; off >= 4; off >>= 1) {
      if (width > 1) {
        const int hw = width / 2;
        const bool upper = (lane & off) != 0;
#pragma unroll
        for (int j = 0; j < GLA_COLS / 2; j++) {
          if (j < hw) {
            const float send = upper ? o[j] : o[j + hw];
            const float keep = upper ? o[j + hw] : o[j];
            o[j] = keep + __shfl_xor_sync(THA_FULL_MASK, send, off);
          }
        }
        width = hw;
      } else {
        o[0] += __shfl_xor_sync(THA_FULL_MASK, o[0], off);
      }
    }
    o[0] += __shfl_xor_sync(THA_FULL_MASK, o[0], 2);
    o[0] += __shfl_xor_sync(THA_FULL_MASK, o[0], 1);
    {
      constexpr int LG = GLA_COLS == 8 ? 3 : GLA_COLS == 4 ? 2 : GLA_COLS == 2 ? 1 : 0;
      const int col = LG ? (lane >> (5 - LG)) : 0;                 // the column this lane ended with
      const bool writer = (lane & ((32 >> LG) - 1)) == 0;
      if (writer && e0 + col < E) o_raw[(size_t)r * g.heads * E + (size_t)h * E + e0 + col] = o[0];
    }
  };
  // whole groups without a branch between their tokens (the refill row is clamped instead of tested), then the ragged end
  int rb = r_begin;
  for (; rb + AHEAD <= r_end; rb += AHEAD) {
#pragma unroll
    for (int u = 0; u < AHEAD; u++) token(rb + u, ring[u], min(rb + u + AHEAD, r_end - 1));
  }
#pragma unroll
  for (int u = 0; u < AHEAD; u++)
    if (rb + u < r_end) token(rb + u, ring[u], -1);
  if (LOCAL) {
    leave(segs.states + (size_t)(at.entry + at.seg) * entry + mine);
    if (e0 == 0) {
#pragma unroll
      for (int i = 0; i < RPL; i++)
        if (ch(i) < D) segs.prods[(size_t)(at.entry + at.seg) * g.heads * D + h * D + ch(i)] = prod[i];
    }
  } else if (at.seg == at.n_seg - 1) {
    leave(slot);
  }
}

// end states from zero -> true end states, a thread per state element of a head, the segments in order (eight loads in flight)
__global__ void hyb_scan_combine_kernel(tha_gla_t g, tha_rows_t rows, ScanSegs segs) {
  const int EP = (g.vdim + GLA_STATE_PAD - 1) / GLA_STATE_PAD * GLA_STATE_PAD, n = g.dim * EP;
  const int i = blockIdx.x * blockDim.x + threadIdx.x, h = blockIdx.y, s = blockIdx.z;
  if (i >= n) return;
  int entry = 0, n_seg = 0;
  for (int t = 0; t <= s; t++) {
    entry += n_seg;
    const int len = rows.seq_first[t + 1] - rows.seq_first[t];
    n_seg = len > segs.len ? (len + segs.len - 1) / segs.len : 0;
  }
  if (n_seg < 3) return;                       // the first segment's end state is true already
  const int d = (i % (2 * g.dim)) >> 1;
  const size_t pitch = (size_t)g.heads * n, ppitch = (size_t)g.heads * g.dim;
  float* S = segs.states + (size_t)entry * pitch + (size_t)h * n + i;
  const float* P = segs.prods + (size_t)entry * ppitch + h * g.dim + d;
  float run = S[0];
  for (int k0 = 1; k0 < n_seg - 1; k0 += 8) {
    float v[8], p[8];
#pragma unroll
    for (int j = 0; j < 8; j++)
      if (k0 + j < n_seg - 1) { v[j] = S[(size_t)(k0 + j) * pitch]; p[j] = P[(size_t)(k0 + j) * ppitch]; }
#pragma unroll
    for (int j = 0; j < 8; j++)
      if (k0 + j < n_seg - 1) { run = fmaf(p[j], run, v[j]); S[(size_t)(k0 + j) * pitch] = run; }
  }
}

}  // namespace tha

using namespace tha;

// THA_SCAN_SEGMENTS=0 runs every portion as one segment (A/B aid)
static bool scan_segments_on() {
  static int on = -1;
  if (on < 0) { const char* v = getenv("THA_SCAN_SEGMENTS"); on = (v && *v) ? atoi(v) != 0 : 1; }
  return on != 0;
}
static int scan_segment_len(int n_rows) {   // at most 32 segments' worth of rows, no segment under 64 rows
  const int len = (n_rows + 31) / 32;
  return len < 64 ? 64 : (len + 15) / 16 * 16;
}
static long long scan_max_segments(int n_rows, int n_seqs) {   // of portions longer than a segment: each has at most 2 n / len
  const long long len = scan_segment_len(n_rows), a = 2ll * n_rows / len, b = n_rows / len + n_seqs;
  return a < b ? a : b;
}

// the scan over decays and inputs that are ready: q at o_q, k at o_k, v at o_v of proj, the read-out times qscale
template <int FORM>
static int gla_scan_launch(cudaStream_t s, const tha_gla_t* g, const tha_rows_t* rows, const tha_state_store_t* st, const float* proj,
                           long long ldp, const float* dec, const float* aux, float* o_raw, float qscale, float* scratch, size_t scratch_floats) {
  constexpr int LFORM = FORM == SCAN_HEAD_DECAY ? SCAN_HEAD_DECAY : SCAN_CHANNEL_DECAY;
  // Segments pay where one portion is much longer than the step's work spread over the machine (about four warps of two columns per
  // scheduler): then the scan is a chain of dependent instructions with idle schedulers beside it.
  ScanSegs segs = {};
  const int len = scan_segment_len(rows->n_rows);
  const double spread = (double)rows->n_rows * g->heads * ceil_div(g->vdim, 2) / (148.0 * 16.0);
  if (scratch && scan_segments_on() && rows->max_seq_rows >= 3 * len && rows->max_seq_rows > 1.5 * spread) {
    const long long n = scan_max_segments(rows->n_rows, rows->n_seqs);
    const size_t state = (size_t)tha_hyb_scan_state_floats(g->heads, g->dim, g->vdim);
    if (n * (state + (size_t)g->heads * g->dim) <= scratch_floats) {
      segs.len = len; segs.states = scratch; segs.prods = scratch + n * state;
    }
  }
  const bool seg = segs.len > 0;
  const int vec = g->dim <= 32 ? 1 : g->dim <= 64 ? 2 : 4;
  const bool wide = seg && g->dim > 32 && g->dim <= 128 && g->dim % vec == 0 && g->o_q % vec == 0 && g->o_k % vec == 0 && ldp % 4 == 0 && g->o_v % 4 == 0 &&
                    g->vdim % 4 == 0 && aligned16(proj) && (!dec || aligned16(dec));
  const bool decode = !seg && rows->max_seq_rows <= 2 && g->dim <= 128;
  const int cols = wide ? 8 : (seg || decode) && g->dim <= 128 ? 4 : 2;
  const dim3 grid(seg ? rows->n_rows / len + rows->n_seqs : rows->n_seqs, g->heads, ceil_div(g->vdim, cols * GLA_WARPS)), block(32 * GLA_WARPS);
#define GLA_LAUNCH(R, A, C, F, L, V) THA_CUDA_OK(launch(hyb_gla_scan_kernel<R, A, C, F, L, V>, grid, block, 0, s, false, *g, *rows, *st, proj, ldp, dec, aux, o_raw, qscale, segs))
#define GLA_BOTH(R, A, C, V) do { if (seg) { GLA_LAUNCH(R, A, C, LFORM, true, V); \
    THA_CUDA_OK(launch(hyb_scan_combine_kernel, dim3(ceil_div(g->dim * ((g->vdim + GLA_STATE_PAD - 1) / GLA_STATE_PAD * GLA_STATE_PAD), 256), g->heads, rows->n_seqs), \
                       dim3(256), 0, s, false, *g, *rows, segs)); } \
    GLA_LAUNCH(R, A, C, FORM, false, V); } while (0)
  // many warps per scheduler (segments): wide loads, eight columns a warp, two tokens ahead; few: two columns, four tokens ahead
  if (wide) { if (g->dim <= 64) GLA_BOTH(2, 2, 8, 2); else GLA_BOTH(4, 2, 8, 4); }
  // decoding: nearly all of it is reading and writing states, so many warps with few registers each
  else if (decode) { if (g->dim <= 32) GLA_LAUNCH(1, 1, 4, FORM, false, 1); else if (g->dim <= 64) GLA_LAUNCH(2, 1, 4, FORM, false, 1); else GLA_LAUNCH(4, 1, 4, FORM, false, 1); }
  else if (g->dim <= 32) { if (cols == 4) GLA_BOTH(1, 4, 4, 1); else GLA_BOTH(1, 4, 2, 1); }
  else if (g->dim <= 64) { if (cols == 4) GLA_BOTH(2, 4, 4, 1); else GLA_BOTH(2, 4, 2, 1); }
  else if (g->dim <= 128) { if (cols == 4) GLA_BOTH(4, 4, 4, 1); else GLA_BOTH(4, 4, 2, 1); }
  else if (g->dim <= 256) GLA_BOTH(8, 2, 2, 1);
  else GLA_BOTH(16, 1, 2, 1);
#undef GLA_BOTH
#undef GLA_LAUNCH
  return THA_STATUS_SUCCESS;
}

extern "C" size_t tha_hyb_scan_scratch_floats(int heads, int dim, int vdim, int n_rows, int n_seqs, int max_seq_rows) {
  if (max_seq_rows < 3 * scan_segment_len(n_rows)) return 0;
  return (size_t)scan_max_segments(n_rows, n_seqs) * (size_t)(tha_hyb_scan_state_floats(heads, dim, vdim) + (long long)heads * dim);
}

namespace tha {
int hyb_scan_launch(cudaStream_t s, int form, const tha_gla_t* g, const tha_rows_t* rows, const tha_state_store_t* st, const float* proj, long long ldp,
                    const float* dec, const float* aux, float* o_raw, float qscale, float* scratch, size_t scratch_floats) {
  if (form == SCAN_HEAD_DECAY) return gla_scan_launch<SCAN_HEAD_DECAY>(s, g, rows, st, proj, ldp, dec, aux, o_raw, qscale, scratch, scratch_floats);
  if (form == SCAN_BONUS) return gla_scan_launch<SCAN_BONUS>(s, g, rows, st, proj, ldp, dec, aux, o_raw, qscale, scratch, scratch_floats);
  return gla_scan_launch<SCAN_CHANNEL_DECAY>(s, g, rows, st, proj, ldp, dec, aux, o_raw, qscale, scratch, scratch_floats);
}
}  // namespace tha

extern "C" long long tha_hyb_scan_state_floats(int heads, int dim, int vdim) {
  return (long long)heads * dim * ((vdim + GLA_STATE_PAD - 1) / GLA_STATE_PAD * GLA_STATE_PAD);
}

extern "C" int tha_hyb_gla_scan(void* stream, int dtype, const tha_gla_t* g, const tha_rows_t* rows, const tha_state_store_t* st,
                                const float* proj, long long ldp, float* z_raw, float* o_raw, void* out, float* seg_scratch, size_t seg_scratch_floats) {
  if (rows->n_seqs < 1 || rows->n_rows < 1) return THA_STATUS_SUCCESS;
  if (g->heads < 1 || g->dim < 1 || g->vdim < 1 || !(g->tau > 0.f)) return THA_STATUS_INVALID_ARG;
  if (g->dim > 512) return THA_STATUS_NOT_SUPPORTED;   // 16 key channels per lane is the widest register form
  cudaStream_t s = (cudaStream_t)stream;
  const size_t n = (size_t)rows->n_rows * g->heads * g->dim;
  THA_CUDA_OK(launch(hyb_gla_decay_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, false, z_raw, n, g->heads * g->dim, g->b_a2,
                     1.0f / g->tau));
  const int status = hyb_scan_launch(s, SCAN_CHANNEL_DECAY, g, rows, st, proj, ldp, z_raw, nullptr, o_raw, 1.0f / sqrtf((float)g->dim), seg_scratch,
                                     seg_scratch_floats);
  if (status != THA_STATUS_SUCCESS) return status;
  return tha_hyb_head_gate(stream, dtype, out, o_raw, rows->n_rows, g->heads, g->vdim, 1, g->eps, g->norm, 0, proj + g->o_g, ldp, THA_GATE_SILU);
}

// The bounded-forget-gate recurrence (tha_hgrn_t) is the same scan with k = 1 - f and a = f.  Its gate arithmetic runs for all
// rows at once, in place: q -> silu(q), the f columns -> 1 - f (what is written), decay <- f = lower + (1 - lower) sigmoid(z + b).
// 1 - f is formed as (1 - lower) (1 - sigmoid(z + b)) so that a nearly closed gate keeps its relative precision.
extern "C" int tha_hyb_hgrn_scan(void* stream, int dtype, const tha_hgrn_t* g, const tha_rows_t* rows, const tha_state_store_t* st,
                                 float* proj, long long ldp, float* decay, float* o_raw, void* out, float* seg_scratch, size_t seg_scratch_floats) {
  if (rows->n_seqs < 1 || rows->n_rows < 1) return THA_STATUS_SUCCESS;
  if (g->heads < 1 || g->dim < 1 || g->vdim < 1) return THA_STATUS_INVALID_ARG;
  if (g->dim > 512) return THA_STATUS_NOT_SUPPORTED;
  cudaStream_t s = (cudaStream_t)stream;
  const size_t n = (size_t)rows->n_rows * g->heads * g->dim;
  THA_CUDA_OK(launch(hyb_hgrn_gates_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, false, proj, ldp, decay, n, g->heads * g->dim,
                     g->o_q, g->o_f, g->f_b, g->lower));
  tha_gla_t a = {};
  a.heads = g->heads; a.dim = g->dim; a.vdim = g->vdim; a.o_q = g->o_q; a.o_k = g->o_f; a.o_v = g->o_v; a.state_off = g->state_off;
  const int status = hyb_scan_launch(s, SCAN_CHANNEL_DECAY, &a, rows, st, proj, ldp, decay, nullptr, o_raw, 1.0f, seg_scratch, seg_scratch_floats);
  if (status != THA_STATUS_SUCCESS) return status;
  return tha_hyb_head_gate(stream, dtype, out, o_raw, rows->n_rows, g->heads, g->vdim, 1, g->eps, g->norm, 0, nullptr, 0, THA_GATE_SIGMOID);
}

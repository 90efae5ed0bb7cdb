// linrec.cu — linear recurrences with a diagonal decay, for the layers of a model given as a list
// (nvllm_mixer_kind NVLLM_MIXER_GLA and the time-mixing side of NVLLM_MIXER_ATTN_TMIX).
//
// Per head a dim x vdim state S in fp32, zero at a sequence's start, kept per state slot:
//   gated linear attention   a_t = sigmoid(z_t)^(1 / tau),  S <- diag(a_t) S + k_t v_t^T,  o_t = S^T q_t
//   time mixing              w_t = exp(-exp(z_t)),  o_t = (S + diag(u) k_t v_t^T)^T r_t,  S <- diag(w_t) S + k_t v_t^T
//   HGRN2                    f_t = l + (1 - l) sigmoid(z_t),  S <- diag(f_t) S + (1 - f_t) v_t^T,  o_t = S^T silu(q_t)
//   mLSTM                    S <- a_t S + b_t k_t v_t^T,  n <- a_t n + b_t k_t,  o_t = S^T q_t / (max(|n . q_t|, c_t) + 1e-6)
//                            a_t = exp(f_t + m_(t-1) - m_t), b_t = exp(i_t - m_t), c_t = exp(-m_t), m_t = max(f_t + m_(t-1), i_t)
// with z_t = W_2 f(W_1 x_t) + b per (head, key entry): f = identity / tanh.  The decay rows belong to
// key entries.  (HGRN2: z_t = W_f x_t + b, one projection, and the
// gate also is the key.)  The read-out of a head is divided by its root mean square, multiplied by a weight
// and (HGRN2: not) by silu(gate) and goes to the output projection.  mLSTM: one forget and one input gate per head,
// given as logarithms f_t = log sigmoid(g(z)), i_t = g(z), g(z) = cap tanh(z / cap); S and n are kept relative to the
// running maximum m_t (0 before the first token); weight per entry of all heads, sigmoid(gate).
//
//   linrec_prep_kernel   per tile of tokens: split-K sums of the projections, q scaled, the second step of
//                        the decay's projection (fp32 FMA, the inner size is small) and the decay itself —
//                        logarithms, exponentials and sigmoids in fp32 (log-sigmoid form, no overflow).
//   hgrn_prep_kernel     HGRN2's epilogue: silu(q), the bounded gate and its complement (neither by a
//                        subtraction from one: both sides of the sigmoid come from one exponential).
//   mlstm_prep_kernel    mLSTM's: the gates' logarithms and the running maximum, which is a scan over the tokens (the
//                        pairs (sum of f, maximum) compose associatively: no long sums of f are subtracted), a | b | c.
//   linrec_scan_kernel   CTA = (sequence, head, range of value columns).  The state sits in registers, a tile of
//                        8 rows by CN columns per lane, updated with packed fp32 instructions.  Token inputs are
//                        staged through shared memory in chunks, the next chunk's loads in flight (cp.async)
//                        while the current one is scanned; the row groups' partial read-outs meet by
//                        shuffles, the warps' in shared memory once per chunk.  State read from the slot when the
//                        sequence has earlier tokens, written back at the end.
//   linrec_out_kernel    per token, a warp per head: RMS over vdim, weight, silu(gate) -> act dtype.
//   linrec_decode_kernel steps with one row per sequence (decode): the three kernels above as one launch per layer.
//   token_shift_kernel   the inputs of time mixing's projections: h_t + (h_{t-1} - h_t) mu_s.
//   roll_tails_kernel    after a step, the last inputs of a short convolution / token shift become
//                        the slot's tail (one thread per channel reads all it needs, then writes).
#include <stdlib.h>

#include <algorithm>

#include "common.cuh"
#include "kernels.h"
#include "mma.cuh"
#include "moe_route.cuh"

namespace nvllm {

namespace {
__device__ __forceinline__ int lr_seq_of_row(const int* __restrict__ cu_q, int n_seqs, int row) {
  int lo = 0, hi = n_seqs - 1;  // last s with cu_q[s] <= row
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= row) lo = mid;
    else hi = mid - 1;
  }
  return lo;
}
__device__ __forceinline__ float seg_at(const LinSeg& g, int t, int c) {
  const float* p = g.p + (size_t)t * g.ld + c;
  float acc = 0.f;
  for (int s = 0; s < g.S; s++) acc += p[(size_t)s * g.stride];
  return acc;
}
// q, k and v projections that came out as one slice each need no summing: the scan reads them
// where the GEMMs left them and the prep kernel writes only the decay
__host__ __device__ __forceinline__ bool linrec_direct(const LinRecArgs& a) { return a.q.S == 1 && a.k.S == 1 && a.v.S == 1; }
__device__ __forceinline__ void lr_cp_async4(uint32_t dst, const void* src, bool ok) {
  const int n = ok ? 4 : 0;  // src-size 0: the destination is filled with zeros
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
}  // namespace

// ------------------------------------------------------------------ projections' epilogue
// grid (ceil(T / TT), Y), 256 threads: a CTA takes TT tokens, a thread one of the H * dim key
// entries at a time.  Output: qkw rows [q | k | decay] and vv (q unscaled: the scan scales its read-outs).  The entry's row of the decay's second-step matrix is read once (16 floats
// at a time, in registers) for all TT tokens, whose inner vectors sit in shared memory and are
// read as broadcasts — the matrix crosses L2 once per TT tokens instead of once per token.
constexpr int LP_RC = 16;  // inner entries per register chunk

template <int TT>
__global__ void __launch_bounds__(256) linrec_prep_kernel(LinRecArgs a, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  extern __shared__ __align__(16) float lr[];  // [TT][rank_p], rank_p = rank rounded up to LP_RC, zero padded
  pdl_wait();
  const int t0 = blockIdx.x * TT;
  const int nt = min(TT, a.T - t0);
  const int rank_p = (a.rank + LP_RC - 1) / LP_RC * LP_RC;
  const int hd = a.H * a.dim, hv = a.H * a.vdim;
  for (int i = threadIdx.x; i < TT * rank_p; i += blockDim.x) {
    const int tt = i / rank_p, r = i % rank_p;
    float x = 0.f;
    if (tt < nt && r < a.rank) {
      x = seg_at(a.lr, t0 + tt, r);
      if (a.tmix) x = tanhf(x);
    }
    lr[i] = x;
  }
  __syncthreads();
  const float inv_tau = 1.0f / a.tau;
  const bool vec_ok = (a.rank % 4) == 0;
  const bool direct = linrec_direct(a);
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < hd; c += gridDim.y * blockDim.x) {
    const float* w = a.w2 + (size_t)c * a.rank;
    float z[TT];
#pragma unroll
    for (int tt = 0; tt < TT; tt++) z[tt] = 0.f;
    for (int r0 = 0; r0 < a.rank; r0 += LP_RC) {
      float wr[LP_RC];
      if (vec_ok && r0 + LP_RC <= a.rank) {
#pragma unroll
        for (int q = 0; q < LP_RC / 4; q++) {
          const float4 v = *reinterpret_cast<const float4*>(w + r0 + 4 * q);
          wr[4 * q] = v.x; wr[4 * q + 1] = v.y; wr[4 * q + 2] = v.z; wr[4 * q + 3] = v.w;
        }
      } else {
#pragma unroll
        for (int q = 0; q < LP_RC; q++) wr[q] = r0 + q < a.rank ? w[r0 + q] : 0.f;
      }
#pragma unroll
      for (int tt = 0; tt < TT; tt++) {
        const float* l = lr + tt * rank_p + r0;
#pragma unroll
        for (int q = 0; q < LP_RC / 4; q++) {
          const float4 v = *reinterpret_cast<const float4*>(l + 4 * q);
          z[tt] = fmaf(wr[4 * q], v.x, z[tt]);
          z[tt] = fmaf(wr[4 * q + 1], v.y, z[tt]);
          z[tt] = fmaf(wr[4 * q + 2], v.z, z[tt]);
          z[tt] = fmaf(wr[4 * q + 3], v.w, z[tt]);
        }
      }
    }
    const float b = a.w2b[c];
    float qv[TT], kv[TT];
    if (!direct) {  // all the loads first
#pragma unroll
      for (int tt = 0; tt < TT; tt++)
        if (tt < nt) {
          qv[tt] = seg_at(a.q, t0 + tt, c);
          kv[tt] = seg_at(a.k, t0 + tt, c);
        }
    }
#pragma unroll
    for (int tt = 0; tt < TT; tt++) {
      if (tt >= nt) break;
      const float zz = z[tt] + b;
      float decay;
      if (a.tmix) {
        decay = expf(-expf(zz));
      } else {
        // sigmoid(z)^(1 / tau) = exp(log sigmoid(z) / tau), log sigmoid(z) = min(z, 0) - log1p(exp(-|z|))
        const float ls = fminf(zz, 0.f) - log1pf(expf(-fabsf(zz)));
        decay = expf(ls * inv_tau);
      }
      float* qkw = a.qkw + (size_t)(t0 + tt) * 3 * hd;
      if (!direct) {
        qkw[c] = qv[tt];
        qkw[hd + c] = kv[tt];
      }
      qkw[2 * hd + c] = decay;
    }
  }
  if (direct) return;
  for (int tt = 0; tt < nt; tt++) {
    float* vv = a.vv + (size_t)(t0 + tt) * hv;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < hv; c += gridDim.y * blockDim.x) vv[c] = seg_at(a.v, t0 + tt, c);
  }
  TRACE_EXIT(tr);
}

cudaError_t launch_linrec_prep(cudaStream_t st, const LinRecArgs& a) {
  if (a.T <= 0) return cudaSuccess;
  const int big = std::max(a.H * a.dim, a.H * a.vdim);
  const int rank_p = (a.rank + LP_RC - 1) / LP_RC * LP_RC;
  if (a.T >= 2048) {
    const size_t smem = (size_t)16 * rank_p * sizeof(float);
    if (smem > 48 * 1024) cudaFuncSetAttribute(linrec_prep_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    (void)launch_k(linrec_prep_kernel<16>, dim3(ceil_div(a.T, 16), std::min(4, ceil_div(big, 256))), dim3(256), smem, st, a,
                   next_trace(40));
  } else if (a.T >= 512) {
    const size_t smem = (size_t)4 * rank_p * sizeof(float);
    if (smem > 48 * 1024) cudaFuncSetAttribute(linrec_prep_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    (void)launch_k(linrec_prep_kernel<4>, dim3(ceil_div(a.T, 4), std::min(8, ceil_div(big, 256))), dim3(256), smem, st, a,
                   next_trace(40));
  } else {  // decode-sized steps: latency matters, not the matrix's trips through L2 — a CTA per token and 256 entries
    const size_t smem = (size_t)rank_p * sizeof(float);
    if (smem > 48 * 1024) cudaFuncSetAttribute(linrec_prep_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    (void)launch_k(linrec_prep_kernel<1>, dim3(a.T, std::min(16, ceil_div(big, 256))), dim3(256), smem, st, a, next_trace(40));
  }
  return cudaGetLastError();
}

// f = l + (1 - l) sigmoid(z) and 1 - f = (1 - l) sigmoid(-z)
__device__ __forceinline__ void bounded_gate(float z, float l, float* f, float* w) {
  const float e = expf(-fabsf(z)), big = 1.0f / (1.0f + e), small = e * big;
  *f = fmaf(1.0f - l, z >= 0.f ? big : small, l);
  *w = (1.0f - l) * (z >= 0.f ? small : big);
}

// grid (T, Y), a thread per VEC neighbouring key entries (VEC = 4: 16-byte accesses; every row must allow them)
template <int VEC>
__global__ void __launch_bounds__(256) hgrn_prep_kernel(LinRecArgs a, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, hd = a.H * a.dim, hv = a.H * a.vdim;
  auto take = [&](const LinSeg& g, int c, float (&v)[VEC]) {
    const float* p = g.p + (size_t)t * g.ld + c;
    if constexpr (VEC == 4) {
      float4 x = *reinterpret_cast<const float4*>(p);
      for (int s = 1; s < g.S; s++) {
        const float4 y = *reinterpret_cast<const float4*>(p + (size_t)s * g.stride);
        x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
      }
      v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    } else {
      v[0] = seg_at(g, t, c);
    }
  };
  auto put = [&](float* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
  };
  float* qkw = a.qkw + (size_t)t * 3 * hd;
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; c < hd; c += gridDim.y * blockDim.x * VEC) {
    float q[VEC], z[VEC], k[VEC], f[VEC];
    take(a.q, c, q);
    take(a.lr, c, z);
#pragma unroll
    for (int e = 0; e < VEC; e++) {
      bounded_gate(z[e] + a.w2b[c + e], a.lower[c + e], &f[e], &k[e]);
      q[e] = silu(q[e]);
    }
    put(qkw + c, q);
    put(qkw + hd + c, k);
    put(qkw + 2 * hd + c, f);
  }
  if (a.v.S > 1)
    for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; c < hv; c += gridDim.y * blockDim.x * VEC) {
      float v[VEC];
      take(a.v, c, v);
      put(a.vv + (size_t)t * hv + c, v);
    }
  TRACE_EXIT(tr);
}

cudaError_t launch_hgrn_prep(cudaStream_t st, const LinRecArgs& a) {
  if (a.T <= 0) return cudaSuccess;
  if (!a.lower) return cudaErrorInvalidValue;
  const int hd = a.H * a.dim, hv = a.H * a.vdim;
  auto ok = [](const LinSeg& g) { return g.ld % 4 == 0 && g.stride % 4 == 0 && reinterpret_cast<size_t>(g.p) % 16 == 0; };
  const bool vec = hd % 4 == 0 && hv % 4 == 0 && ok(a.q) && ok(a.lr) && ok(a.v);
  const int per = 256 * (vec ? 4 : 1);
  const dim3 grid(a.T, a.T >= 1024 ? 1 : std::min(8, ceil_div(std::max(hd, hv), per)));
  const int threads = std::min(256, std::max(32, ceil_div(ceil_div(std::max(hd, hv), vec ? 4 : 1), 32) * 32));
  if (vec) (void)launch_k(hgrn_prep_kernel<4>, grid, dim3(threads), 0, st, a, next_trace(40));
  else (void)launch_k(hgrn_prep_kernel<1>, grid, dim3(threads), 0, st, a, next_trace(40));
  return cudaGetLastError();
}

// ---- mLSTM
__device__ __forceinline__ void mlstm_log_gates(float zi, float zf, float cap, float* gi, float* gf) {
  *gi = cap * tanhf(zi / cap);
  const float x = cap * tanhf(zf / cap);
  *gf = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));  // log sigmoid(x)
}
// The first n_seqs * H CTAs: one (sequence, head) each, 256 tokens at a time.  Token t takes the running maximum m to
// max(m + F, I) with (F, I) = (f_t, i_t), and two such steps compose to (F1 + F2, max(I1 + F2, I2)): a warp scans its 32
// tokens by shuffles, the warps' totals meet in shared memory.  The others sum q, k and v's slices (none when direct).
constexpr int MP_NT = 256;
__global__ void __launch_bounds__(MP_NT) mlstm_prep_kernel(LinRecArgs a, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  pdl_wait();
  const int n_gate = a.n_seqs * a.H;
  if ((int)blockIdx.x >= n_gate) {
    const int hd = a.H * a.dim, hv = a.H * a.vdim;
    for (int t = blockIdx.x - n_gate; t < a.T; t += gridDim.x - n_gate) {
      float* qkw = a.qkw + (size_t)t * 3 * hd;
      for (int c = threadIdx.x; c < hd; c += MP_NT) {
        qkw[c] = seg_at(a.q, t, c);
        qkw[hd + c] = seg_at(a.k, t, c);
      }
      for (int c = threadIdx.x; c < hv; c += MP_NT) a.vv[(size_t)t * hv + c] = seg_at(a.v, t, c);
    }
    TRACE_EXIT(tr);
    return;
  }
  __shared__ float sF[MP_NT / 32], sI[MP_NT / 32], s_last;
  const int seq = blockIdx.x / a.H, head = blockIdx.x % a.H;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int r0 = a.cu_q[seq], n_new = a.cu_q[seq + 1] - r0;
  if (n_new <= 0) return;
  float* top = a.state_pool + (size_t)a.state_slots[seq] * a.slot_floats + a.max_off + head;
  float m0 = a.positions[r0] > 0 ? *top : 0.f;
  const size_t plane = (size_t)a.T * a.H;
  for (int t0 = 0; t0 < n_new; t0 += MP_NT) {
    const int t = t0 + threadIdx.x;
    const bool ok = t < n_new;
    float gi = -INFINITY, gf = 0.f;
    if (ok) mlstm_log_gates(seg_at(a.gi, r0 + t, head) + a.gi_b[head], seg_at(a.gf, r0 + t, head) + a.gf_b[head], a.cap, &gi, &gf);
    float F = gf, I = gi;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float F1 = __shfl_up_sync(0xffffffffu, F, o), I1 = __shfl_up_sync(0xffffffffu, I, o);
      if (lane >= o) {
        I = fmaxf(I1 + F, I);
        F += F1;
      }
    }
    if (lane == 31) {
      sF[warp] = F;
      sI[warp] = I;
    }
    __syncthreads();
    float base = m0;  // the maximum before the warp's first token
    for (int w = 0; w < warp; w++) base = fmaxf(base + sF[w], sI[w]);
    const float m = fmaxf(base + F, I);
    float prev = __shfl_up_sync(0xffffffffu, m, 1);
    if (lane == 0) prev = base;
    if (ok) {
      float* g = a.gates + (size_t)(r0 + t) * a.H + head;
      g[0] = expf(gf + prev - m);
      g[plane] = expf(gi - m);
      g[2 * plane] = expf(-m);
    }
    if (threadIdx.x == MP_NT - 1) s_last = m;  // (tokens past the end leave the maximum as it is)
    __syncthreads();
    m0 = s_last;
  }
  if (threadIdx.x == 0) *top = m0;
  TRACE_EXIT(tr);
}

cudaError_t launch_mlstm_prep(cudaStream_t st, const LinRecArgs& a) {
  if (a.T <= 0) return cudaSuccess;
  if (!a.gi.p || !a.gf.p || !a.gates || !(a.cap > 0.f)) return cudaErrorInvalidValue;
  const int sums = linrec_direct(a) ? 0 : std::min(a.T, 148 * 8);
  (void)launch_k(mlstm_prep_kernel, dim3(a.n_seqs * a.H + sums), dim3(MP_NT), 0, st, a, next_trace(40));
  return cudaGetLastError();
}

// ------------------------------------------------------------------ scan over tokens
// A lane holds a tile of the state, 8 rows (four packed pairs of neighbouring rows) by CN value columns, in
// registers; a warp covers 8 RG rows by (32 / RG) CN columns, a CTA's WR warps the rows of the head.  Per token a
// lane reads its 8 entries of q, k and decay and its CN values (16-byte shared-memory loads, broadcast among the
// lanes that share them) for 8 CN state entries, and updates two rows with one packed fp32 instruction
// (f32x2: two independent IEEE fp32 operations).  The row groups' partial read-outs are summed by shuffles that
// scatter the columns over the lanes, the warps' in shared memory once per chunk of tokens.
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ unsigned long long mul2(unsigned long long a, unsigned long long b) {
  unsigned long long d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ unsigned long long pack2(float lo, float hi) {
  unsigned long long d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ void unpack2(unsigned long long v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}

// DP: rows of the state, padded (RG * 8 * WR); TMIX: read before the update, with a bonus; SD: one decay per
// (token, head) instead of one per row; NRM (with SD): mLSTM — keys are scaled by the token's input gate, and the CTAs of
// the first column range carry the vector n beside the state (every column group of lanes holds its 8 entries)
template <int RG, int WR, int CN, bool TMIX, bool SD, bool NRM>
__global__ void __launch_bounds__(32 * WR) linrec_scan_kernel(LinRecArgs a, int vec16, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  constexpr int NT = 32 * WR, CG = 32 / RG, DP = 8 * RG * WR, VC = CG * CN;
  constexpr int TC = DP >= 256 ? 4 : 8;                        // tokens per staged chunk
  constexpr int ROW = 3 * DP + VC;                             // floats of one staged token: q | k | decay | v
  constexpr int NO = CN >= RG ? CN / RG : 1;                   // columns a lane holds after the shuffles
  __shared__ __align__(16) float stage[2][TC][ROW];
  __shared__ float part[WR][TC][VC];
  __shared__ float part_n[NRM ? WR : 1][TC];
  const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * VC;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rg = lane / CG, cg = lane % CG;
  const int row0 = (warp * RG + rg) * 8;                       // this lane's first row
  const int dim = a.dim, vdim = a.vdim, hd = a.H * dim, hv = a.H * vdim;
  pdl_wait();
  const int r0 = a.cu_q[seq], n_new = a.cu_q[seq + 1] - r0;
  if (n_new <= 0) return;
  const bool has_prev = a.positions[r0] > 0;
  float* state = a.state_pool + (size_t)a.state_slots[seq] * a.slot_floats + a.state_off + (size_t)head * dim * vdim;

  // q | k | decay | v of the step's rows: the projections' own output when it needs no summing
  const bool direct = linrec_direct(a);
  const int qk_head = a.qk_div > 1 ? head / a.qk_div : head;
  const float* part_p[3] = {(direct ? a.q.p : a.qkw) + qk_head * dim, (direct ? a.k.p : a.qkw + hd) + qk_head * dim,
                            SD ? a.decay_p + head : a.qkw + 2 * hd + head * dim};
  const size_t part_ld[3] = {direct ? (size_t)a.q.ld : (size_t)3 * hd, direct ? (size_t)a.k.ld : (size_t)3 * hd,
                             SD ? (size_t)a.decay_ld : (size_t)3 * hd};
  const float* v_p = (direct ? a.v.p : a.vv) + head * vdim + col0;
  const size_t v_ld = direct ? (size_t)a.v.ld : (size_t)hv;
  auto load_chunk = [&](int t0, int buf) {
    const int nt = min(TC, n_new - t0);
    if (vec16) {  // every row, head and column range starts on a 16-byte boundary and is whole 16-byte pieces long
      constexpr int NP = SD ? 2 : 3;
#pragma unroll
      for (int pt = 0; pt < NP; pt++)
        for (int i = tid; i < TC * (DP / 4); i += NT) {
          const int tt = i / (DP / 4), r = (i % (DP / 4)) * 4;
          const bool ok = tt < nt && r < dim;
          cp_async16(smem_addr(&stage[buf][tt][pt * DP + r]), part_p[pt] + (size_t)(r0 + t0 + (ok ? tt : 0)) * part_ld[pt] + (ok ? r : 0), ok);
        }
      for (int i = tid; i < TC * (VC / 4); i += NT) {
        const int tt = i / (VC / 4), c = (i % (VC / 4)) * 4;
        const bool ok = tt < nt && col0 + c < vdim;
        cp_async16(smem_addr(&stage[buf][tt][3 * DP + c]), v_p + (size_t)(r0 + t0 + (ok ? tt : 0)) * v_ld + (ok ? c : 0), ok);
      }
    } else {
      for (int i = tid; i < TC * 3 * DP; i += NT) {
        const int tt = i / (3 * DP), j = i % (3 * DP), pt = j / DP, r = j % DP;
        if (SD && pt == 2) continue;
        const bool ok = tt < nt && r < dim;
        lr_cp_async4(smem_addr(&stage[buf][tt][j]), part_p[pt] + (size_t)(r0 + t0 + (ok ? tt : 0)) * part_ld[pt] + (ok ? r : 0), ok);
      }
      for (int i = tid; i < TC * VC; i += NT) {
        const int tt = i / VC, c = i % VC;
        const bool ok = tt < nt && col0 + c < vdim;
        lr_cp_async4(smem_addr(&stage[buf][tt][3 * DP + c]), v_p + (size_t)(r0 + t0 + (ok ? tt : 0)) * v_ld + (ok ? c : 0), ok);
      }
    }
    if (SD)
      for (int tt = tid; tt < TC; tt += NT) {
        const size_t t = r0 + t0 + (tt < nt ? tt : 0);
        lr_cp_async4(smem_addr(&stage[buf][tt][2 * DP]), part_p[2] + t * part_ld[2], tt < nt);
        if (NRM) lr_cp_async4(smem_addr(&stage[buf][tt][2 * DP + 1]), a.gates + ((size_t)a.T + t) * a.H + head, tt < nt);
      }
  };
  load_chunk(0, 0);
  cp_async_commit();

  unsigned long long S[4][CN], U[TMIX ? 4 : 1];
#pragma unroll
  for (int p = 0; p < 4; p++) {
    float s[2][CN];
#pragma unroll
    for (int e = 0; e < 2; e++)
#pragma unroll
      for (int c = 0; c < CN; c++) {
        const int r = row0 + 2 * p + e, col = col0 + cg * CN + c;
        s[e][c] = (r < dim && col < vdim && has_prev) ? state[(size_t)r * vdim + col] : 0.f;
      }
#pragma unroll
    for (int c = 0; c < CN; c++) S[p][c] = pack2(s[0][c], s[1][c]);
    if (TMIX) {
      const int r = row0 + 2 * p;
      U[p] = pack2(r < dim ? a.bonus[head * dim + r] : 0.f, r + 1 < dim ? a.bonus[head * dim + r + 1] : 0.f);
    }
  }

  const bool with_n = NRM && blockIdx.z == 0;
  float* nvec = NRM ? a.state_pool + (size_t)a.state_slots[seq] * a.slot_floats + a.norm_off + (size_t)head * dim : nullptr;
  unsigned long long N[NRM ? 4 : 1];
  if (NRM)
#pragma unroll
    for (int p = 0; p < 4; p++) {
      const int r = row0 + 2 * p;
      N[NRM ? p : 0] = pack2(with_n && has_prev && r < dim ? nvec[r] : 0.f, with_n && has_prev && r + 1 < dim ? nvec[r + 1] : 0.f);
    }

  const int n_chunks = (n_new + TC - 1) / TC;
  for (int ch = 0; ch < n_chunks; ch++) {
    const int buf = ch & 1;
    if (ch + 1 < n_chunks) load_chunk((ch + 1) * TC, buf ^ 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const int nt = min(TC, n_new - ch * TC);
#pragma unroll 2
    for (int tt = 0; tt < nt; tt++) {
      const float* row = stage[buf][tt];
      unsigned long long q[4], k[4], w[4], acc[CN];
      float v[CN];
#pragma unroll
      for (int p = 0; p < 2; p++) {
        const ulonglong2 x = *reinterpret_cast<const ulonglong2*>(row + row0 + 4 * p);
        const ulonglong2 y = *reinterpret_cast<const ulonglong2*>(row + DP + row0 + 4 * p);
        q[2 * p] = x.x; q[2 * p + 1] = x.y;
        k[2 * p] = y.x; k[2 * p + 1] = y.y;
        if (!SD) {
          const ulonglong2 z = *reinterpret_cast<const ulonglong2*>(row + 2 * DP + row0 + 4 * p);
          w[2 * p] = z.x; w[2 * p + 1] = z.y;
        }
      }
      if (SD) {
        const float d = row[2 * DP];
        w[0] = w[1] = w[2] = w[3] = pack2(d, d);
      }
      if (NRM) {
        const float b = row[2 * DP + 1];
        const unsigned long long bb = pack2(b, b);
#pragma unroll
        for (int p = 0; p < 4; p++) k[p] = mul2(k[p], bb);
        if (with_n) {
          unsigned long long ac = 0ull;
#pragma unroll
          for (int p = 0; p < 4; p++) {
            N[NRM ? p : 0] = fma2(w[p], N[NRM ? p : 0], k[p]);
            ac = fma2(q[p], N[NRM ? p : 0], ac);
          }
          float lo, hi;
          unpack2(ac, lo, hi);
          float s = lo + hi;
#pragma unroll
          for (int off = 16; off >= CG; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
          if (lane == 0) part_n[NRM ? warp : 0][tt] = s;
        }
      }
      const float* vr = row + 3 * DP + cg * CN;
      if constexpr (CN >= 4) {
#pragma unroll
        for (int c = 0; c < CN; c += 4) {
          const float4 x = *reinterpret_cast<const float4*>(vr + c);
          v[c] = x.x; v[c + 1] = x.y; v[c + 2] = x.z; v[c + 3] = x.w;
        }
      } else {
#pragma unroll
        for (int c = 0; c < CN; c++) v[c] = vr[c];
      }
#pragma unroll
      for (int c = 0; c < CN; c++) {
        const unsigned long long vd = pack2(v[c], v[c]);
        unsigned long long ac = 0ull;  // (+0, +0)
#pragma unroll
        for (int p = 0; p < 4; p++) {
          const unsigned long long kv = mul2(k[p], vd);
          if (TMIX) {
            ac = fma2(q[p], fma2(U[p], kv, S[p][c]), ac);
            S[p][c] = fma2(w[p], S[p][c], kv);
          } else {
            S[p][c] = fma2(w[p], S[p][c], kv);
            ac = fma2(q[p], S[p][c], ac);
          }
        }
        acc[c] = ac;
      }
      float o[CN];
#pragma unroll
      for (int c = 0; c < CN; c++) {
        float lo, hi;
        unpack2(acc[c], lo, hi);
        o[c] = lo + hi;
      }
      // sum over the row groups: every exchange halves the columns a lane is responsible for
      int n = CN, cofs = 0;
#pragma unroll
      for (int off = 16; off >= CG; off >>= 1) {
        if (n > 1) {
          n >>= 1;
          const bool up = lane & off;
#pragma unroll
          for (int i = 0; i < CN / 2; i++)
            if (i < n) {
              const float send = up ? o[i] : o[i + n], mine = up ? o[i + n] : o[i];
              o[i] = mine + __shfl_xor_sync(0xffffffffu, send, off);
            }
          cofs += up ? n : 0;
        } else {
          o[0] += __shfl_xor_sync(0xffffffffu, o[0], off);
        }
      }
#pragma unroll
      for (int i = 0; i < NO; i++) part[warp][tt][cg * CN + cofs + i] = o[i];
    }
    __syncthreads();  // the warps' partial read-outs are in; the staged chunk has been consumed
    for (int i = tid; i < nt * VC; i += NT) {
      const int tt = i / VC, c = i % VC;
      float t = 0.f;
#pragma unroll
      for (int w = 0; w < WR; w++) t += part[w][tt][c];
      if (col0 + c < vdim) a.o[(size_t)(r0 + ch * TC + tt) * hv + head * vdim + col0 + c] = t * a.qmul;
    }
    if (with_n)
      for (int tt = tid; tt < nt; tt += NT) {
        float t = 0.f;
#pragma unroll
        for (int w = 0; w < WR; w++) t += part_n[NRM ? w : 0][tt];
        a.nq[(size_t)(r0 + ch * TC + tt) * a.H + head] = t * a.qmul;
      }
  }
  cp_async_wait<0>();
  if (with_n && cg == 0)
#pragma unroll
    for (int p = 0; p < 4; p++) {
      float lo, hi;
      unpack2(N[NRM ? p : 0], lo, hi);
      const int r = row0 + 2 * p;
      if (r < dim) nvec[r] = lo;
      if (r + 1 < dim) nvec[r + 1] = hi;
    }
#pragma unroll
  for (int p = 0; p < 4; p++)
#pragma unroll
    for (int c = 0; c < CN; c++) {
      float lo, hi;
      unpack2(S[p][c], lo, hi);
      const int r = row0 + 2 * p, col = col0 + cg * CN + c;
      if (r < dim && col < vdim) state[(size_t)r * vdim + col] = lo;
      if (r + 1 < dim && col < vdim) state[(size_t)(r + 1) * vdim + col] = hi;
    }
  TRACE_EXIT(tr);
}

template <int RG, int WR, int CN>
static cudaError_t linrec_scan_launch_cn(cudaStream_t st, const LinRecArgs& a) {
  const dim3 grid(a.n_seqs, a.H, ceil_div(a.vdim, 32 / RG * CN));
  auto ok = [](const void* p, size_t ld) { return reinterpret_cast<size_t>(p) % 16 == 0 && ld % 4 == 0; };
  const int hd = a.H * a.dim;
  bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0;
  if (linrec_direct(a)) vec = vec && ok(a.q.p, a.q.ld) && ok(a.k.p, a.k.ld) && ok(a.v.p, a.v.ld);
  else vec = vec && ok(a.qkw, 3 * (size_t)hd) && ok(a.vv, (size_t)a.H * a.vdim);
  if (!a.decay_p) vec = vec && ok(a.qkw, 3 * (size_t)hd);
  const int v16 = vec ? 1 : 0;
  if (a.gi.p) (void)launch_k(linrec_scan_kernel<RG, WR, CN, false, true, true>, grid, dim3(32 * WR), 0, st, a, v16, next_trace(41));
  else if (a.tmix) (void)launch_k(linrec_scan_kernel<RG, WR, CN, true, false, false>, grid, dim3(32 * WR), 0, st, a, v16, next_trace(41));
  else if (a.decay_p) (void)launch_k(linrec_scan_kernel<RG, WR, CN, false, true, false>, grid, dim3(32 * WR), 0, st, a, v16, next_trace(41));
  else (void)launch_k(linrec_scan_kernel<RG, WR, CN, false, false, false>, grid, dim3(32 * WR), 0, st, a, v16, next_trace(41));
  return cudaGetLastError();
}
template <int RG, int WR>
static cudaError_t linrec_scan_launch(cudaStream_t st, const LinRecArgs& a) {
  // four columns per lane (eight were slower: too few warps to cover the latency of a token); a sequence's tokens
  // are scanned in order, so few long sequences want narrower, more CTAs
  constexpr int CG = 32 / RG;
  const long units = (long)a.n_seqs * a.H;
  if (a.vdim > CG * 2 && units * ceil_div(a.vdim, CG * 4) >= 148) return linrec_scan_launch_cn<RG, WR, 4>(st, a);
  return linrec_scan_launch_cn<RG, WR, 2>(st, a);
}

cudaError_t launch_linrec_scan(cudaStream_t st, const LinRecArgs& a) {
  if (a.T <= 0 || a.n_seqs <= 0) return cudaSuccess;
  if (a.dim > LINREC_MAX_DIM || (a.tmix && !a.bonus) || (a.gi.p && (!a.decay_p || !a.gates || !a.nq))) return cudaErrorInvalidValue;
  if (a.dim <= 16) return linrec_scan_launch<2, 1>(st, a);
  if (a.dim <= 32) return linrec_scan_launch<4, 1>(st, a);
  if (a.dim <= 64) return linrec_scan_launch<4, 2>(st, a);
  if (a.dim <= 128) return linrec_scan_launch<4, 4>(st, a);
  return linrec_scan_launch<4, 8>(st, a);
}

// ------------------------------------------------------------------ one token per sequence: everything in one kernel
// A decode step gives every sequence one row, and a head whose value columns fit one CTA
// (vdim <= 32 CC) needs nothing from other CTAs: the projections' epilogue (split-K sums, the
// decay), the state update with its read-out, the head's RMS norm, weight and gate run as ONE
// launch per layer instead of three.  CTA = (sequence, head); the state slice of a thread is as
// in linrec_scan_kernel and its loads are in flight while the row's inputs are prepared.
// KIND: 0 gated linear attention, 1 time mixing, 2 HGRN2, 3 mLSTM
template <int RPL, int NW, int CC, int KIND>
__global__ void __launch_bounds__(32 * NW) linrec_decode_kernel(LinRecArgs a, int out_bf16, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  constexpr bool TMIX = KIND == 1;
  constexpr int NT = 32 * NW;
  constexpr int DP = RPL * NW;
  constexpr int VC = 32 * CC;
  extern __shared__ __align__(16) float sm[];
  float* sq = sm;                 // [DP] q | [DP] k | [DP] decay
  float* sv = sm + 3 * DP;        // [VC]
  float* part = sv + VC;          // [NW][VC]
  float* slr = part + NW * VC;    // [rank]
  __shared__ float red[32];
  __shared__ float s_gate[3];     // mLSTM: a | b | c
  const int t = blockIdx.x, head = blockIdx.y;
  const int tid = threadIdx.x, l = tid >> 5, lane = tid & 31;
  const int dim = a.dim, vdim = a.vdim;
  pdl_wait();
  const bool has_prev = a.positions[t] > 0;
  float* state = a.state_pool + (size_t)a.state_slots[t] * a.slot_floats + a.state_off + (size_t)head * dim * vdim;
  float S[CC][RPL], U[TMIX ? RPL : 1];
#pragma unroll
  for (int g = 0; g < RPL / 4; g++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int r = (g * NW + l) * 4 + e;
#pragma unroll
      for (int cc = 0; cc < CC; cc++) {
        const int col = cc * 32 + lane;
        S[cc][g * 4 + e] = (r < dim && col < vdim && has_prev) ? state[(size_t)r * vdim + col] : 0.f;
      }
      if (TMIX) U[g * 4 + e] = r < dim ? a.bonus[head * dim + r] : 0.f;
    }
  for (int r = tid; r < a.rank; r += NT) {
    const float x = seg_at(a.lr, t, r);
    slr[r] = a.tmix ? tanhf(x) : x;
  }
  for (int c = tid; c < VC; c += NT) sv[c] = c < vdim ? seg_at(a.v, t, head * vdim + c) : 0.f;
  float* slot = a.state_pool + (size_t)a.state_slots[t] * a.slot_floats;
  if (KIND == 3 && tid == 0) {
    float gi, gf;
    mlstm_log_gates(seg_at(a.gi, t, head) + a.gi_b[head], seg_at(a.gf, t, head) + a.gf_b[head], a.cap, &gi, &gf);
    float* top = slot + a.max_off + head;
    const float prev = has_prev ? *top : 0.f, m = fmaxf(gf + prev, gi);
    *top = m;
    s_gate[0] = expf(gf + prev - m);
    s_gate[1] = expf(gi - m);
    s_gate[2] = expf(-m);
  }
  __syncthreads();
  const float inv_tau = 1.0f / a.tau;
  float nq = 0.f;
  for (int i = tid; i < DP; i += NT) {
    float q = 0.f, k = 0.f, decay = 0.f;
    if (KIND == 3) {
      if (i < dim) {
        const int c = head * dim + i;
        float* nvec = slot + a.norm_off + c;
        const float n0 = has_prev ? *nvec : 0.f;
        q = seg_at(a.q, t, c);
        k = seg_at(a.k, t, c) * s_gate[1];
        decay = s_gate[0];
        const float n1 = fmaf(decay, n0, k);
        *nvec = n1;
        nq = fmaf(n1, q, nq);
      }
    } else if (KIND == 2) {
      if (i < dim) {
        const int c = head * dim + i;
        bounded_gate(seg_at(a.lr, t, c) + a.w2b[c], a.lower[c], &decay, &k);
        q = silu(seg_at(a.q, t, c));
      }
    } else if (i < dim) {
      const int c = head * dim + i;
      const float* w = a.w2 + (size_t)c * a.rank;
      float z = 0.f;
      if ((a.rank & 3) == 0) {  // 16-byte loads of the matrix row, four at a time in flight
#pragma unroll 4
        for (int r = 0; r < a.rank; r += 4) {
          const float4 wv = *reinterpret_cast<const float4*>(w + r);
          z = fmaf(wv.x, slr[r], z);
          z = fmaf(wv.y, slr[r + 1], z);
          z = fmaf(wv.z, slr[r + 2], z);
          z = fmaf(wv.w, slr[r + 3], z);
        }
      } else {
        for (int r = 0; r < a.rank; r++) z = fmaf(w[r], slr[r], z);
      }
      z += a.w2b[c];
      if (a.tmix) {
        decay = expf(-expf(z));
      } else {
        const float ls = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));  // log sigmoid(z)
        decay = expf(ls * inv_tau);
      }
      q = seg_at(a.q, t, c);
      k = seg_at(a.k, t, c);
    }
    sq[i] = q;
    sq[DP + i] = k;
    sq[2 * DP + i] = decay;
  }
  __syncthreads();
  float v[CC], acc[CC];
#pragma unroll
  for (int cc = 0; cc < CC; cc++) {
    v[cc] = sv[cc * 32 + lane];
    acc[cc] = 0.f;
  }
#pragma unroll
  for (int g = 0; g < RPL / 4; g++) {
    const int rb = (g * NW + l) * 4;
    const float4 q4 = *reinterpret_cast<const float4*>(sq + rb);
    const float4 k4 = *reinterpret_cast<const float4*>(sq + DP + rb);
    const float4 w4 = *reinterpret_cast<const float4*>(sq + 2 * DP + rb);
    const float qq[4] = {q4.x, q4.y, q4.z, q4.w}, kk[4] = {k4.x, k4.y, k4.z, k4.w}, ww[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
    for (int e = 0; e < 4; e++) {
#pragma unroll
      for (int cc = 0; cc < CC; cc++) {
        float& st = S[cc][g * 4 + e];
        if (TMIX) {
          const float kv = kk[e] * v[cc];
          acc[cc] = fmaf(qq[e], fmaf(U[g * 4 + e], kv, st), acc[cc]);
          st = fmaf(ww[e], st, kv);
        } else {
          st = fmaf(ww[e], st, kk[e] * v[cc]);
          acc[cc] = fmaf(qq[e], st, acc[cc]);
        }
      }
    }
  }
#pragma unroll
  for (int cc = 0; cc < CC; cc++) part[l * VC + cc * 32 + lane] = acc[cc];
#pragma unroll
  for (int g = 0; g < RPL / 4; g++)
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int r = (g * NW + l) * 4 + e;
#pragma unroll
      for (int cc = 0; cc < CC; cc++) {
        const int col = cc * 32 + lane;
        if (r < dim && col < vdim) state[(size_t)r * vdim + col] = S[cc][g * 4 + e];
      }
    }
  __syncthreads();
  // the head's read-out: a thread per column (NT >= 128 >= VC)
  float o = 0.f, gt = 0.f, wn = 0.f;
  const bool mine = tid < vdim;
  if (mine) {
#pragma unroll
    for (int w = 0; w < NW; w++) o += part[w * VC + tid];
    o *= a.qmul;
    if (KIND != 2) gt = seg_at(a.gate, t, head * vdim + tid);
    wn = a.onorm_w[(size_t)head * a.onorm_ld + tid];
  }
  if (KIND == 3) o /= fmaxf(fabsf(block_sum(nq, red) * a.qmul), s_gate[2]) + 1e-6f;
  const float inv = 1.0f / sqrtf(block_sum(o * o, red) / (float)vdim + a.eps);
  const float res = KIND == 2 ? o * inv * wn : o * inv * wn * (KIND == 3 ? 1.0f / (1.0f + expf(-gt)) : silu(gt));
  if (out_bf16) {
    bf16* out = (bf16*)a.out + (size_t)t * a.o_ld;
    if (mine) out[head * vdim + tid] = __float2bfloat16_rn(res);
    if (head == 0)
      for (int c = a.H * vdim + tid; c < a.o_ld; c += NT) out[c] = __float2bfloat16_rn(0.f);
  } else {
    float* out = (float*)a.out + (size_t)t * a.o_ld;
    if (mine) out[head * vdim + tid] = res;
    if (head == 0)
      for (int c = a.H * vdim + tid; c < a.o_ld; c += NT) out[c] = 0.f;
  }
  TRACE_EXIT(tr);
}

template <int RPL, int NW, int CC>
static cudaError_t linrec_decode_launch_cc(cudaStream_t st, int odt, const LinRecArgs& a) {
  const size_t smem = (size_t)(3 * RPL * NW + 32 * CC + NW * 32 * CC + a.rank) * sizeof(float);
  const int bf = odt == DT_BF16;
#define LD(KIND_)                                                                                                        \
  do {                                                                                                                   \
    if (smem > 48 * 1024)                                                                                                \
      cudaFuncSetAttribute(linrec_decode_kernel<RPL, NW, CC, KIND_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    (void)launch_k(linrec_decode_kernel<RPL, NW, CC, KIND_>, dim3(a.T, a.H), dim3(32 * NW), smem, st, a, bf, next_trace(45)); \
  } while (0)
  if (a.gi.p) LD(3);
  else if (a.lower) LD(2);
  else if (a.tmix) LD(1);
  else LD(0);
#undef LD
  return cudaGetLastError();
}
template <int RPL, int NW>
static cudaError_t linrec_decode_launch(cudaStream_t st, int odt, const LinRecArgs& a) {
  if (a.vdim <= 32) return linrec_decode_launch_cc<RPL, NW, 1>(st, odt, a);
  if (a.vdim <= 64) return linrec_decode_launch_cc<RPL, NW, 2>(st, odt, a);
  return linrec_decode_launch_cc<RPL, NW, 4>(st, odt, a);
}
bool linrec_decode_fused_ok(const LinRecArgs& a) {
  static const bool on = [] {
    const char* e = getenv("NVLLM_LINREC_FUSED");
    return e ? atoi(e) != 0 : true;
  }();
  return on && a.T == a.n_seqs && a.vdim <= 128 && a.dim <= LINREC_MAX_DIM;
}
cudaError_t launch_linrec_decode(cudaStream_t st, int odt, const LinRecArgs& a) {
  if (a.T <= 0) return cudaSuccess;
  if (!linrec_decode_fused_ok(a) || (a.tmix && !a.bonus)) return cudaErrorInvalidValue;
  if (a.dim <= 16) return linrec_decode_launch<4, 4>(st, odt, a);
  if (a.dim <= 32) return linrec_decode_launch<8, 4>(st, odt, a);
  if (a.dim <= 64) return linrec_decode_launch<16, 4>(st, odt, a);
  if (a.dim <= 128) return linrec_decode_launch<32, 4>(st, odt, a);
  return linrec_decode_launch<32, 8>(st, odt, a);
}

// ------------------------------------------------------------------ gated norm of the read-out
// MJ: 16-byte pieces per lane (vdim <= 128 MJ); GATED: 0 no gate, 1 silu(gate), 2 mLSTM: the read-out is first divided by
// max(|n . q|, c) + 1e-6, sigmoid(gate)
template <int GATED>
__device__ __forceinline__ float out_gate(float z) { return GATED == 2 ? 1.0f / (1.0f + expf(-z)) : silu(z); }
template <typename OT, int MJ, int GATED>
__global__ void __launch_bounds__(256) linrec_out_kernel(LinRecArgs a, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const int vdim = a.vdim;
  OT* out = (OT*)a.out + (size_t)t * a.o_ld;
  // 16-byte loads when every row and head starts on a 16-byte boundary
  const bool vec = (vdim % 4) == 0 && vdim <= 128 * MJ && (a.gate.ld % 4) == 0 && (a.gate.stride % 4) == 0 &&
                   (reinterpret_cast<size_t>(a.gate.p) % 16) == 0 && (a.onorm_ld % 4) == 0;
  for (int h = blockIdx.y * nw + warp; h < a.H; h += gridDim.y * nw) {
    const float* o = a.o + (size_t)t * a.H * vdim + (size_t)h * vdim;
    float od = 1.f;  // what the read-out is divided by
    if (GATED == 2) od = fmaxf(fabsf(a.nq[(size_t)t * a.H + h]), a.gates[((size_t)2 * a.T + t) * a.H + h]) + 1e-6f;
    if (vec) {
      // four neighbouring columns per lane, all loads (read-outs, gate slices, weights) before the arithmetic
      float4 ov[MJ], gv[GATED ? MJ : 1];
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < MJ; j++) {
        const int i = lane * 4 + 128 * j;
        if (i < vdim) {
          ov[j] = *reinterpret_cast<const float4*>(o + i);
          if constexpr (GATED == 2) { ov[j].x /= od; ov[j].y /= od; ov[j].z /= od; ov[j].w /= od; }
          ss += ov[j].x * ov[j].x + ov[j].y * ov[j].y + ov[j].z * ov[j].z + ov[j].w * ov[j].w;
          if constexpr (GATED) {
            const float* gp = a.gate.p + (size_t)t * a.gate.ld + h * vdim + i;
            gv[j] = *reinterpret_cast<const float4*>(gp);
            for (int sl = 1; sl < a.gate.S; sl++) {
              const float4 x = *reinterpret_cast<const float4*>(gp + (size_t)sl * a.gate.stride);
              gv[j].x += x.x; gv[j].y += x.y; gv[j].z += x.z; gv[j].w += x.w;
            }
          }
        }
      }
      const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + a.eps);
      const float* w = a.onorm_w + (size_t)h * a.onorm_ld;
#pragma unroll
      for (int j = 0; j < MJ; j++) {
        const int i = lane * 4 + 128 * j;
        if (i < vdim) {
          const float4 w4 = *reinterpret_cast<const float4*>(w + i);
          float r[4] = {ov[j].x * inv * w4.x, ov[j].y * inv * w4.y, ov[j].z * inv * w4.z, ov[j].w * inv * w4.w};
          if constexpr (GATED) {
            r[0] *= out_gate<GATED>(gv[j].x); r[1] *= out_gate<GATED>(gv[j].y);
            r[2] *= out_gate<GATED>(gv[j].z); r[3] *= out_gate<GATED>(gv[j].w);
          }
          store4(out + h * vdim + i, r);
        }
      }
      continue;
    }
    float ss = 0.f;
    for (int i = lane; i < vdim; i += 32) ss += (o[i] / od) * (o[i] / od);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + a.eps);
    const float* w = a.onorm_w + (size_t)h * a.onorm_ld;
    for (int i = lane; i < vdim; i += 32) {
      const float r = o[i] / od * inv * w[i];
      out[h * vdim + i] = from_f32<OT>(GATED ? r * out_gate<GATED>(seg_at(a.gate, t, h * vdim + i)) : r);
    }
  }
  if (blockIdx.y == 0)
    for (int c = a.H * vdim + threadIdx.x; c < a.o_ld; c += blockDim.x) out[c] = from_f32<OT>(0.f);
  TRACE_EXIT(tr);
}

cudaError_t launch_linrec_out(cudaStream_t st, int odt, const LinRecArgs& a) {
  if (a.T <= 0) return cudaSuccess;
  const dim3 grid(a.T, a.T >= 1024 ? 1 : ceil_div(a.H, 8));
#define LO(OT_, MJ_)                                                                                           \
  do {                                                                                                         \
    if (a.gi.p) (void)launch_k(linrec_out_kernel<OT_, MJ_, 2>, grid, dim3(256), 0, st, a, next_trace(42));         \
    else if (a.gate.p) (void)launch_k(linrec_out_kernel<OT_, MJ_, 1>, grid, dim3(256), 0, st, a, next_trace(42));  \
    else (void)launch_k(linrec_out_kernel<OT_, MJ_, 0>, grid, dim3(256), 0, st, a, next_trace(42));         \
  } while (0)
  if (odt == DT_F32) {
    if (a.vdim <= 128) LO(float, 1); else LO(float, 4);
  } else {
    if (a.vdim <= 128) LO(bf16, 1); else LO(bf16, 4);
  }
#undef LO
  return cudaGetLastError();
}

// ------------------------------------------------------------------ token shift
template <typename AT>
__global__ void __launch_bounds__(256) token_shift_kernel(int T, int n_seqs, int W, int n_mix, const AT* __restrict__ h,
                                                          const float* __restrict__ mu, const int* __restrict__ cu_q,
                                                          const int* __restrict__ positions,
                                                          const int* __restrict__ state_slots,
                                                          const float* __restrict__ state_pool, size_t slot_floats,
                                                          size_t tail_off, AT* __restrict__ out, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  // the row's sequence: every thread tests one sequence's range (one round trip, no dependent chain)
  __shared__ int s_seq;
  if (T == n_seqs) {
    if (threadIdx.x == 0) s_seq = t;
  } else {
    for (int i = threadIdx.x; i < n_seqs; i += blockDim.x)
      if (cu_q[i] <= t && t < cu_q[i + 1]) s_seq = i;
  }
  __syncthreads();
  const int s = s_seq;
  const int r0 = cu_q[s];
  const bool in_step = t > r0;
  const bool in_slot = !in_step && positions[t] > 0;
  const float* tail = state_pool + (size_t)state_slots[s] * slot_floats + tail_off;
  for (int i = threadIdx.x * 8; i < W; i += blockDim.x * 8) {  // W is a multiple of 8
    float x[8], xp[8];
    load8(h + (size_t)t * W + i, x);
    if (in_step) load8(h + (size_t)(t - 1) * W + i, xp);
    else if (in_slot) load8(tail + i, xp);
    else
#pragma unroll
      for (int e = 0; e < 8; e++) xp[e] = 0.f;
    for (int m = 0; m < n_mix; m++) {
      float w[8], y[8];
      load8(mu + (size_t)m * W + i, w);
#pragma unroll
      for (int e = 0; e < 8; e++) y[e] = fmaf(xp[e] - x[e], w[e], x[e]);
      store8(out + ((size_t)m * T + t) * W + i, y);
    }
  }
  TRACE_EXIT(tr);
}

cudaError_t launch_token_shift(cudaStream_t st, int adt, int T, int n_seqs, int W, int n_mix, const void* h,
                               const float* mu, const int* cu_q, const int* positions, const int* state_slots,
                               const float* state_pool, size_t slot_floats, size_t tail_off, void* out) {
  if (T <= 0) return cudaSuccess;
  if (adt == DT_F32)
    (void)launch_k(token_shift_kernel<float>, dim3(T), dim3(128), 0, st, T, n_seqs, W, n_mix, (const float*)h, mu, cu_q,
                   positions, state_slots, state_pool, slot_floats, tail_off, (float*)out, next_trace(43));
  else
    (void)launch_k(token_shift_kernel<bf16>, dim3(T), dim3(128), 0, st, T, n_seqs, W, n_mix, (const bf16*)h, mu, cu_q,
                   positions, state_slots, state_pool, slot_floats, tail_off, (bf16*)out, next_trace(43));
  return cudaGetLastError();
}

// ------------------------------------------------------------------ convolution on a sublayer's input
// One CTA per token, eight channels per thread; TAPS > 0: the number of taps at compile time.  Where tap
// j's input lives is the same for every channel of the row: a row of this step, a row of the slot's
// tail, or nowhere (before the sequence's start).  With a router the fp32 row is routed here.
template <typename AT, int TAPS>
__global__ void __launch_bounds__(512) input_conv_kernel(InputConvArgs a, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  extern __shared__ __align__(16) float row[];  // [W] with a router
  __shared__ int s_seq;
  constexpr int MT = TAPS > 0 ? TAPS : INPUT_CONV_MAX_TAPS;
  const int taps = TAPS > 0 ? TAPS : a.taps, W = a.W;
  const int t = blockIdx.x;
  // (the step's integer inputs are in place before any kernel of the step starts)
  if (a.T == a.n_seqs) {
    if (threadIdx.x == 0) s_seq = t;
  } else {
    for (int i = threadIdx.x; i < a.n_seqs; i += blockDim.x)
      if (a.cu_q[i] <= t && t < a.cu_q[i + 1]) s_seq = i;
  }
  __syncthreads();
  const int s = s_seq;
  const int li = t - a.cu_q[s], pos = a.positions[t], keep = taps - 1;
  const float* tail = taps > 1 ? a.state_pool + (size_t)a.state_slots[s] * a.slot_floats + a.tail_off : nullptr;
  const float* src[MT];
#pragma unroll
  for (int j = 0; j < MT; j++) {
    src[j] = nullptr;
    if (j < taps) {
      const int back = keep - j;  // input `back` positions before this token
      if (back <= li) src[j] = a.h + (size_t)(t - back) * W;
      else if (back <= pos) src[j] = tail + (size_t)(keep - (back - li)) * W;
    }
  }
  pdl_wait();
  for (int c = threadIdx.x * 8; c < W; c += blockDim.x * 8) {
    float y[8];
    if constexpr (TAPS > 0) {
      float u[MT][8], wv[MT][8];
#pragma unroll
      for (int j = 0; j < MT; j++) {  // all the loads first
        if (src[j]) load8(src[j] + c, u[j]);
        else
#pragma unroll
          for (int e = 0; e < 8; e++) u[j][e] = 0.f;
        load8(a.w + (size_t)j * W + c, wv[j]);
      }
#pragma unroll
      for (int e = 0; e < 8; e++) y[e] = u[MT - 1][e];
#pragma unroll
      for (int j = 0; j < MT; j++)
#pragma unroll
        for (int e = 0; e < 8; e++) y[e] = fmaf(wv[j][e], u[j][e], y[e]);
    } else {
      load8(a.h + (size_t)t * W + c, y);
#pragma unroll
      for (int j = 0; j < MT; j++)
        if (j < taps && src[j]) {
          float u[8], wv[8];
          load8(src[j] + c, u);
          load8(a.w + (size_t)j * W + c, wv);
#pragma unroll
          for (int e = 0; e < 8; e++) y[e] = fmaf(wv[e], u[e], y[e]);
        }
    }
    store8((AT*)a.out + (size_t)t * W + c, y);
    if (a.router) store8(row + c, y);
  }
  if (a.router) {
    __shared__ float probs[MOE_MAX_E];
    __syncthreads();
    moe_route_row(row, a.router, W, a.E, a.topk, probs, (size_t)t, a.topk_idx, a.topk_w, a.route);
  }
  TRACE_EXIT(tr);
}

// The same for steps of many rows with a router: a CTA takes TT tokens, their convolved rows stay in
// shared memory and are routed together (moe_route_tile).
template <typename AT, int TAPS, int TT>
__global__ void __launch_bounds__(256) input_conv_route_kernel(InputConvArgs a, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  extern __shared__ __align__(16) float rows[];  // [TT][W], then probs | chs | gsc [TT][E] each
  __shared__ int s_seq[TT];
  const int W = a.W, E = a.E, t0 = blockIdx.x * TT, nt = min(TT, a.T - t0), keep = a.taps - 1;
  const int warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  for (int i = threadIdx.x; i < a.n_seqs; i += blockDim.x) {
    const int lo = max(a.cu_q[i], t0), hi = min(a.cu_q[i + 1], t0 + nt);
    for (int t = lo; t < hi; t++) s_seq[t - t0] = i;
  }
  __syncthreads();
  pdl_wait();
  const int vpr = W / 8;
  for (int it = threadIdx.x; it < TT * vpr; it += blockDim.x) {
    const int tt = it / vpr, c = (it % vpr) * 8;
    float y[8];
    if (tt < nt) {
      const int t = t0 + tt, s = s_seq[tt], li = t - a.cu_q[s], pos = a.positions[t];
      load8(a.h + (size_t)t * W + c, y);
#pragma unroll
      for (int j = 0; j < (TAPS > 0 ? TAPS : INPUT_CONV_MAX_TAPS); j++) {
        if (TAPS == 0 && j >= a.taps) break;
        const int back = keep - j;
        float u[8], wv[8];
        if (back <= li) load8(a.h + (size_t)(t - back) * W + c, u);
        else if (back <= pos)
          load8(a.state_pool + (size_t)a.state_slots[s] * a.slot_floats + a.tail_off + (size_t)(keep - (back - li)) * W + c, u);
        else continue;
        load8(a.w + (size_t)j * W + c, wv);
#pragma unroll
        for (int e = 0; e < 8; e++) y[e] = fmaf(wv[e], u[e], y[e]);
      }
      store8((AT*)a.out + (size_t)t * W + c, y);
    } else {
#pragma unroll
      for (int e = 0; e < 8; e++) y[e] = 0.f;
    }
    store8(rows + (size_t)tt * W + c, y);
  }
  __syncthreads();
  float* probs = rows + (size_t)TT * W;
  moe_route_tile<TT>(rows, W, a.router, E, a.route.bias, probs);
  __syncthreads();
  for (int tt = warp; tt < nt; tt += nw)
    moe_select_row(probs + tt * E, probs + (size_t)(TT + tt) * E, probs + (size_t)(2 * TT + tt) * E, E, a.topk, (size_t)(t0 + tt),
                   a.topk_idx, a.topk_w, a.route);
  TRACE_EXIT(tr);
}

constexpr int IC_TT = 8;             // tokens per CTA of input_conv_route_kernel
constexpr size_t IC_SMEM = 96 * 1024;  // ... as long as their rows fit (two CTAs per SM)

template <typename AT, int TAPS>
static void input_conv_route(cudaStream_t st, const InputConvArgs& a, size_t smem) {
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(input_conv_route_kernel<AT, TAPS, IC_TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  (void)launch_k(input_conv_route_kernel<AT, TAPS, IC_TT>, dim3(ceil_div(a.T, IC_TT)), dim3(256), smem, st, a, next_trace(43));
}

cudaError_t launch_input_conv(cudaStream_t st, int adt, const InputConvArgs& a) {
  if (a.T <= 0) return cudaSuccess;
  if (a.taps < 1 || a.taps > INPUT_CONV_MAX_TAPS || (a.W & 7)) return cudaErrorInvalidValue;
  int threads = std::min(512, std::max(64, ceil_div(a.W / 8, 32) * 32));
  if (a.router && a.T <= 1024) threads = 512;  // few rows: 16 warps share a row's experts (see launch_norm)
  const size_t tile_smem = ((size_t)IC_TT * a.W + 3 * (size_t)IC_TT * a.E) * sizeof(float);
  if (a.router && a.T >= 1024 && tile_smem <= IC_SMEM) {
    if (adt == DT_F32) {
      if (a.taps == 4) input_conv_route<float, 4>(st, a, tile_smem); else input_conv_route<float, 0>(st, a, tile_smem);
    } else {
      if (a.taps == 4) input_conv_route<bf16, 4>(st, a, tile_smem); else input_conv_route<bf16, 0>(st, a, tile_smem);
    }
    return cudaGetLastError();
  }
  const size_t smem = a.router ? (size_t)a.W * sizeof(float) : 0;
#define IC(AT_, TP_) (void)launch_k(input_conv_kernel<AT_, TP_>, dim3(a.T), dim3(threads), smem, st, a, next_trace(43))
  if (adt == DT_F32) {
    if (a.taps == 2) IC(float, 2); else if (a.taps == 3) IC(float, 3); else if (a.taps == 4) IC(float, 4); else IC(float, 0);
  } else {
    if (a.taps == 2) IC(bf16, 2); else if (a.taps == 3) IC(bf16, 3); else if (a.taps == 4) IC(bf16, 4); else IC(bf16, 0);
  }
#undef IC
  return cudaGetLastError();
}

// ------------------------------------------------------------------ tails of short convolutions
constexpr int TAIL_MAX_TAPS = 8;
struct TailArgs {
  TailJob j[TAIL_MAX_JOBS];
  int n_jobs;
  const int *cu_q, *positions, *state_slots;
  float* state_pool;
  size_t slot_floats;
};
// grid (n_seqs, Y).  Entry i of the new tail is the input at position end - (taps - 1) + i: a row of
// this step, an entry of the old tail, or (before the sequence's start) zero.
template <typename AT>
__global__ void __launch_bounds__(256) roll_tails_kernel(TailArgs a, Trace tr) {
  TRACE_ENTRY(tr);
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.x;
  const int r0 = a.cu_q[s], n_new = a.cu_q[s + 1] - r0;
  if (n_new <= 0) return;
  const int pos0 = a.positions[r0], end = pos0 + n_new;
  float* slot = a.state_pool + (size_t)a.state_slots[s] * a.slot_floats;
  for (int jb = 0; jb < a.n_jobs; jb++) {
    const TailJob& J = a.j[jb];
    const int keep = J.taps - 1;
    float* tail = slot + J.tail_off;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < J.channels; c += gridDim.y * blockDim.x) {
      float nv[TAIL_MAX_TAPS];
#pragma unroll
      for (int i = 0; i < TAIL_MAX_TAPS; i++) {
        nv[i] = 0.f;
        if (i < keep) {
          const int p = end - keep + i;
          if (p >= pos0) {
            const int row = r0 + (p - pos0);
            nv[i] = J.seg.p ? seg_at(J.seg, row, c) + (J.bias ? J.bias[c] : 0.f)
                            : to_f32(((const AT*)J.act)[(size_t)row * J.channels + c]);
          } else if (p >= 0) {
            nv[i] = tail[(size_t)(p - pos0 + keep) * J.channels + c];
          }
        }
      }
#pragma unroll
      for (int i = 0; i < TAIL_MAX_TAPS; i++)
        if (i < keep) tail[(size_t)i * J.channels + c] = nv[i];
    }
  }
  TRACE_EXIT(tr);
}

cudaError_t launch_roll_tails(cudaStream_t st, int adt, int n_seqs, const TailJob* jobs, int n_jobs, const int* cu_q,
                              const int* positions, const int* state_slots, float* state_pool, size_t slot_floats) {
  if (n_seqs <= 0 || n_jobs <= 0) return cudaSuccess;
  if (n_jobs > TAIL_MAX_JOBS) return cudaErrorInvalidValue;
  TailArgs a{};
  int big = 0;
  for (int i = 0; i < n_jobs; i++) {
    if (jobs[i].taps > TAIL_MAX_TAPS) return cudaErrorInvalidValue;
    a.j[i] = jobs[i];
    big = std::max(big, jobs[i].channels);
  }
  a.n_jobs = n_jobs; a.cu_q = cu_q; a.positions = positions; a.state_slots = state_slots;
  a.state_pool = state_pool; a.slot_floats = slot_floats;
  const dim3 grid(n_seqs, std::max(1, std::min(16, ceil_div(big, 256))));
  if (adt == DT_F32) (void)launch_k(roll_tails_kernel<float>, grid, dim3(256), 0, st, a, next_trace(44));
  else (void)launch_k(roll_tails_kernel<bf16>, grid, dim3(256), 0, st, a, next_trace(44));
  return cudaGetLastError();
}

}  // namespace nvllm

// moe_route.cuh — one token's expert routing (moe.go:63-103), shared by the stand-alone router
// kernel (moe.cu) and the norm kernel that fuses it (elementwise.cu).
#pragma once
#include "common.cuh"
#include "kernels.h"

namespace nvllm {

constexpr int MOE_MAX_E = 256;

// ONE warp: from the logits in probs (overwritten) the softmax over ALL E experts
// (tensor.go:128-155), k rounds of first-max selection (ties -> lower index, which is what a
// stable descending sort gives; the reference's sort.Slice is unstable, ties have measure zero
// with random-init weights) and the renormalisation over the chosen k (moe.go:88-103).
// probs, chs, gsc: shared scratch of E floats each, this warp's own.  identity_w (shared): receives the summed weight of
// the chosen identity experts (RouteOpts::identity).
__device__ __forceinline__ void moe_select_row(float* probs, float* chs, float* gsc, int E, int k, size_t t,
                                               int* __restrict__ topk_idx, float* __restrict__ topk_w,
                                               RouteOpts ro, float* identity_w = nullptr) {
  const int lane = threadIdx.x & 31;
  if (ro.sigmoid) {
    // every expert scores on its own
    for (int e = lane; e < E; e += 32) probs[e] = 1.0f / (1.0f + expf(-probs[e]));
    __syncwarp();
  } else {
    float mx = -INFINITY;
    for (int e = lane; e < E; e += 32) mx = fmaxf(mx, probs[e]);
    mx = warp_max(mx);
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) {
      float p = expf(probs[e] - mx);
      probs[e] = p;
      sum += p;
    }
    sum = warp_sum(sum);
    __syncwarp();
    for (int e = lane; e < E; e += 32) probs[e] = probs[e] / sum;
    __syncwarp();
  }
  // The choice may go by other numbers than the weights: ch[e] = probs[e] + correction[e] (any sign;
  // an expert taken out of the choice is -inf), while the weights stay probs[e].
  const bool corr = ro.correction != nullptr;
  float* ch = corr ? chs : probs;
  const float OUT = corr ? -INFINITY : -2.f;   // marks an expert that cannot be chosen (plain scores are >= 0)
  if (corr) {
    for (int e = lane; e < E; e += 32) chs[e] = probs[e] + ro.correction[e];
    __syncwarp();
  }
  // group-limited choice: a group scores as its best expert (or the sum of its two best); group g
  // stays iff fewer than `keep` groups beat it (higher score, or equal score and lower index).
  // Experts of the other groups are taken out of the selection below.
  if (ro.groups > 1 && ro.keep < ro.groups) {
    const int per = E / ro.groups;
    for (int g = lane; g < ro.groups; g += 32) {
      float b1 = -INFINITY, b2 = -INFINITY;
      for (int j = 0; j < per; j++) {
        const float v = ch[g * per + j];
        if (v > b1) { b2 = b1; b1 = v; }
        else if (v > b2) b2 = v;
      }
      gsc[g] = (ro.group_top2 && per > 1) ? b1 + b2 : b1;
    }
    __syncwarp();
    for (int g = lane; g < ro.groups; g += 32) {
      int beat = 0;
      for (int o = 0; o < ro.groups; o++) beat += (gsc[o] > gsc[g] || (gsc[o] == gsc[g] && o < g)) ? 1 : 0;
      if (beat >= ro.keep)
        for (int j = 0; j < per; j++) ch[g * per + j] = OUT;
    }
    __syncwarp();
  }
  float sel_p = 0.f;  // lane s keeps the s-th selection (k <= 32)
  int sel_i = 0;
  float ksum = 0.f;
  for (int s = 0; s < k; s++) {
    float bv = OUT;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      float p = ch[e];
      if (p > bv) {
        bv = p;
        bi = e;
      }
    }
    if (corr) {
      // signed choice scores: order-preserving map of the float's bits to unsigned (-inf lowest)
      const unsigned u = __float_as_uint(bv);
      const unsigned key = (u & 0x80000000u) ? ~u : (u | 0x80000000u);
      const unsigned kmax = __reduce_max_sync(0xffffffffu, key);
      bi = (int)__reduce_min_sync(0xffffffffu, (key == kmax && bi != 0x7fffffff) ? (unsigned)bi : 0x7fffffffu);
      bv = probs[bi];  // the weight comes from the score itself
    } else {
      // warp arg-max in two redux operations instead of five shuffle rounds: probabilities are
      // >= 0, so their bit patterns order like the values (+1 keeps a genuine 0.0 above the -1 of
      // a lane with no candidate); ties go to the lower expert index
      const unsigned key = bv < 0.f ? 0u : __float_as_uint(bv) + 1u;
      const unsigned kmax = __reduce_max_sync(0xffffffffu, key);
      bi = (int)__reduce_min_sync(0xffffffffu, key == kmax ? (unsigned)bi : 0x7fffffffu);
      bv = kmax ? __uint_as_float(kmax - 1u) : -1.f;
    }
    if (lane == s) {
      sel_p = bv;
      sel_i = bi;
    }
    ksum += bv;  // moe.go:98-103: sum in descending order
    if (lane == 0) ch[bi] = OUT;
    __syncwarp();
  }
  if (ro.sigmoid && !ro.raw) ksum += 1e-20f;
  float id_w = 0.f;
  if (lane < k) {
    topk_idx[t * k + lane] = sel_i;
    const float wgt = ro.raw ? sel_p * ro.scale : sel_p / ksum;
    topk_w[t * k + lane] = ro.square ? wgt * wgt : wgt;
    if (sel_i >= E - ro.identity) id_w = wgt;
  }
  if (identity_w) {
    id_w = warp_sum(id_w);
    if (lane == 0) *identity_w = id_w;
  }
}

// All warps of the CTA: warp w computes the logits of experts w, w + nw, ... from the
// normed row y (shared or global memory, fp32) and R [E, H]; warp 0 then selects.
// probs: shared scratch of >= E floats.  Contains __syncthreads.
__device__ __forceinline__ void moe_route_row(const float* y, const float* __restrict__ R, int H,
                                              int E, int k, float* probs, size_t t,
                                              int* __restrict__ topk_idx,
                                              float* __restrict__ topk_w,
                                              RouteOpts ro = RouteOpts{}, float* identity_w = nullptr) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  // Two experts per pass with the k loop unrolled four deep: up to 8 independent 32-byte loads
  // of R per lane in flight, so the E / nw passes cost one L2 round trip each instead of one
  // per 256 columns per expert (measured 10 us per row CTA with the rolled loop at E = 32).
  // The per-expert accumulation order (ascending i, then the warp tree) is unchanged.
  for (int e = warp; e < E; e += 2 * nw) {
    const int e2 = e + nw;
    const bool two = e2 < E;
    const float* r1 = R + (size_t)e * H;
    const float* r2 = R + (size_t)(two ? e2 : e) * H;
    float acc1 = 0.f, acc2 = 0.f;
    for (int i0 = lane * 8; i0 < H; i0 += 1024) {
      float b1[4][8], b2[4][8];
#pragma unroll
      for (int u = 0; u < 4; u++) {
        const int i = i0 + u * 256;
        if (i < H) {
          load8(r1 + i, b1[u]);
          if (two) load8(r2 + i, b2[u]);
        }
      }
#pragma unroll
      for (int u = 0; u < 4; u++) {
        const int i = i0 + u * 256;
        if (i < H) {
          float a[8];
          load8(y + i, a);
#pragma unroll
          for (int j = 0; j < 8; j++) acc1 = fmaf(a[j], b1[u][j], acc1);
          if (two) {
#pragma unroll
            for (int j = 0; j < 8; j++) acc2 = fmaf(a[j], b2[u][j], acc2);
          }
        }
      }
    }
    acc1 = warp_sum(acc1);
    acc2 = warp_sum(acc2);
    if (lane == 0) {
      probs[e] = ro.bias ? acc1 + ro.bias[e] : acc1;
      if (two) probs[e2] = ro.bias ? acc2 + ro.bias[e2] : acc2;
    }
  }
  __syncthreads();
  if (warp != 0) return;
  __shared__ float chs[MOE_MAX_E], gsc[MOE_MAX_E];
  moe_select_row(probs, chs, gsc, E, k, t, topk_idx, topk_w, ro, identity_w);
}

// Router logits of TT rows that sit in shared memory (rows [TT][W], W a multiple of 4): a warp accumulates four experts
// against all of them — a router row crosses L2 once per TT tokens instead of once per token.  probs [TT][E].
template <int TT>
__device__ __forceinline__ void moe_route_tile(const float* rows, int W, const float* __restrict__ R, int E,
                                               const float* __restrict__ bias, float* probs) {
  constexpr int EB = 4;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  for (int e0 = warp * EB; e0 < E; e0 += nw * EB) {
    float acc[EB][TT];
#pragma unroll
    for (int q = 0; q < EB; q++)
#pragma unroll
      for (int tt = 0; tt < TT; tt++) acc[q][tt] = 0.f;
#pragma unroll 2
    for (int i = lane * 4; i < W; i += 128) {  // neighbouring lanes, neighbouring 16-byte pieces: no bank conflicts
      float4 r[EB];
#pragma unroll
      for (int q = 0; q < EB; q++) r[q] = *reinterpret_cast<const float4*>(R + (size_t)min(e0 + q, E - 1) * W + i);
#pragma unroll
      for (int tt = 0; tt < TT; tt++) {
        const float4 y = *reinterpret_cast<const float4*>(rows + (size_t)tt * W + i);
#pragma unroll
        for (int q = 0; q < EB; q++) {
          acc[q][tt] = fmaf(y.x, r[q].x, acc[q][tt]);
          acc[q][tt] = fmaf(y.y, r[q].y, acc[q][tt]);
          acc[q][tt] = fmaf(y.z, r[q].z, acc[q][tt]);
          acc[q][tt] = fmaf(y.w, r[q].w, acc[q][tt]);
        }
      }
    }
#pragma unroll
    for (int q = 0; q < EB; q++)
#pragma unroll
      for (int tt = 0; tt < TT; tt++) {
        const float z = warp_sum(acc[q][tt]);
        if (lane == 0 && e0 + q < E) probs[tt * E + e0 + q] = bias ? z + bias[e0 + q] : z;
      }
  }
}

}  // namespace nvllm

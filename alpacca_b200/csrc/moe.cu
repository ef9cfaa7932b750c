// Routed experts: the router with groups, and the experts' two products for the (token, expert) pairs of a step.
//
// Router, per token, in 32-bit: z = W_r h; s = softmax(z) over all experts; the experts form `groups` equal
// groups of neighbours, a group's score is its largest s, only experts of the `keep` best groups can be
// chosen; the `top` largest s among those are chosen (the lower index wins a tie); their weights are
// s / (sum of the chosen s + 1e-20) * scale.
// Experts: y_t = sum_j weight_j * W_down[e_j] act(W_up[e_j] h_t), act = exact gelu (erf) here.
// Options: a bias on the router's logits; gated experts, y_t = sum_j weight_j * W_down[e_j] (act(W_gate[e_j] h_t) *
// (W_up[e_j] h_t)).  (With one group, all groups kept and scale 1 the weights are the softmax over the chosen
// logits alone: s_j / sum of the chosen s is exp(z_j) / sum of the chosen exp(z).)
// The pair kernels read each chosen expert's rows once per pair: the form for steps of few tokens, where the
// weights stream from memory once and every token adds its experts in the order of its choices.
#include "common.cuh"
#include "launch.cuh"
#include "moe_choice.cuh"

#define MOE_MAX_EXPERTS 1024

// A warp's share of the dot product of two rows of n numbers (add with warp_sum): 16 bytes per lane and
// load where both rows allow it.
__device__ __forceinline__ float lane_dot(const bf16* __restrict__ a, const bf16* __restrict__ b, int n, int lane) {
  float part = 0.f;
  if ((n & 7) == 0 && ((((uintptr_t)a) | ((uintptr_t)b)) & 15) == 0) {
    for (int k = lane * 8; k < n; k += 256) {
      const uint4 x = *reinterpret_cast<const uint4*>(a + k);
      const uint4 y = __ldg(reinterpret_cast<const uint4*>(b + k));
      const __nv_bfloat162* xp = reinterpret_cast<const __nv_bfloat162*>(&x);
      const __nv_bfloat162* yp = reinterpret_cast<const __nv_bfloat162*>(&y);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 xf = __bfloat1622float2(xp[j]), yf = __bfloat1622float2(yp[j]);
        part += xf.x * yf.x + xf.y * yf.y;
      }
    }
    return part;
  }
  for (int k = lane; k < n; k += 32) part += __bfloat162float(a[k]) * __bfloat162float(b[k]);
  return part;
}
__device__ __forceinline__ float lane_dot(const float* __restrict__ a, const float* __restrict__ b, int n, int lane) {
  float part = 0.f;
  for (int k = lane; k < n; k += 32) part += a[k] * b[k];      // one order for every n: the 32-bit path
  return part;
}
__device__ __forceinline__ float lane_dot(const bf16* __restrict__ a, const float* __restrict__ b, int n, int lane) {
  float part = 0.f;
  if ((n & 3) == 0 && (((uintptr_t)a) & 7) == 0 && (((uintptr_t)b) & 15) == 0) {
    for (int k = lane * 4; k < n; k += 128) {
      const uint2 x = *reinterpret_cast<const uint2*>(a + k);
      const float4 y = __ldg(reinterpret_cast<const float4*>(b + k));
      const __nv_bfloat162* xp = reinterpret_cast<const __nv_bfloat162*>(&x);
      const float2 x0 = __bfloat1622float2(xp[0]), x1 = __bfloat1622float2(xp[1]);
      part += x0.x * y.x + x0.y * y.y + x1.x * y.z + x1.y * y.w;
    }
    return part;
  }
  for (int k = lane; k < n; k += 32) part += __bfloat162float(a[k]) * b[k];
  return part;
}

// z[t, e] = W_r[e] . h[t]: one warp per (token, expert)
template <typename T>
__global__ void moe_logits_kernel(const T* __restrict__ h, int ld, const float* __restrict__ wr, int n_tokens, int width,
                                  int E, float* __restrict__ z, const float* __restrict__ bias) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const long long id = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (id >= (long long)n_tokens * E) return;
  const int t = (int)(id / E), e = (int)(id - (long long)t * E);
  const float part = warp_sum(lane_dot(h + (size_t)t * ld, wr + (size_t)e * width, width, lane));
  if (lane == 0) z[id] = part + (bias != nullptr ? bias[e] : 0.f);
}

// z[t, e] alone (float32), without a choice: gate logits of a part that reads the stream
AB_API int ab_moe_logits(const void* h, int dtype, int ld, const float* wr, int n_tokens, int width, int E, float* z,
                         cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  if (E <= 0 || width <= 0) return AB_BAD_ARG;
  const unsigned blocks = (unsigned)(((long long)n_tokens * E + 7) / 8);
  if (dtype == AB_F32)
    ab_launch(moe_logits_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)h, ld, wr, n_tokens, width, E, z, nullptr);
  else if (dtype == AB_BF16)
    ab_launch(moe_logits_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (const bf16*)h, ld, wr, n_tokens, width, E, z, nullptr);
  else
    return AB_BAD_ARG;
  return ab_launch_status();
}

// the choice, one warp per token, from the logits z [T, E]
__global__ void moe_route_kernel(const float* __restrict__ z, int n_tokens, int E, int groups, int keep, int top,
                                 float scale, int* __restrict__ idx, float* __restrict__ wts) {
  extern __shared__ float sm[];           // E scores per warp, then `groups` group scores per warp
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31, wib = threadIdx.x >> 5;
  const int t = blockIdx.x * (blockDim.x >> 5) + wib;
  if (t >= n_tokens) return;
  float* s = sm + (size_t)wib * E;
  for (int e = lane; e < E; e += 32) s[e] = z[(size_t)t * E + e];
  __syncwarp();
  float mx = -INFINITY;
  for (int e = lane; e < E; e += 32) mx = fmaxf(mx, s[e]);
  mx = warp_max(mx);
  float sum = 0.f;
  for (int e = lane; e < E; e += 32) {
    const float p = expf(s[e] - mx);
    s[e] = p;
    sum += p;
  }
  sum = warp_sum(sum);
  __syncwarp();
  for (int e = lane; e < E; e += 32) s[e] = s[e] / sum;
  __syncwarp();
  // groups: the experts of groups that are not kept are struck out (-1, below every score)
  const int per = E / groups;
  if (keep < groups) {
    float* gs = sm + (size_t)(blockDim.x >> 5) * E + (size_t)wib * groups;
    for (int g = lane; g < groups; g += 32) {
      float v = -1.f;
      for (int j = 0; j < per; ++j) v = fmaxf(v, s[g * per + j]);
      gs[g] = v;
    }
    __syncwarp();
    for (int pick = 0; pick < keep; ++pick) {
      float best = -0.5f;
      int bg = 0x7fffffff;
      for (int g = lane; g < groups; g += 32)
        if (gs[g] > best) { best = gs[g]; bg = g; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int og = __shfl_xor_sync(0xffffffffu, bg, o);
        if (ob > best || (ob == best && og < bg)) { best = ob; bg = og; }
      }
      if (lane == 0 && bg != 0x7fffffff) gs[bg] = -2.f;      // kept
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (gs[e / per] != -2.f) s[e] = -1.f;
    __syncwarp();
  }
  float chosen_sum = 0.f;
  for (int pick = 0; pick < top; ++pick) {
    float best = -0.5f;
    int be = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      const float v = s[e];
      if (v > best) { best = v; be = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ob > best || (ob == best && oe < be)) { best = ob; be = oe; }
    }
    if (be == 0x7fffffff) { be = 0; best = 0.f; }      // nothing left to choose (or the row holds no numbers)
    chosen_sum += best;
    if (lane == 0) {
      idx[(size_t)t * top + pick] = be;
      wts[(size_t)t * top + pick] = best;
      s[be] = -1.f;                                    // taken
    }
    __syncwarp();
  }
  if (lane == 0) {
    const float inv = scale / (chosen_sum + 1e-20f);
    for (int j = 0; j < top; ++j) wts[(size_t)t * top + j] *= inv;
  }
}

// `bias`: float [E] added to the logits, or null
AB_API int ab_moe_route_bias(const void* h, int dtype, int ld, const float* wr, const float* bias, int n_tokens, int width,
                             int E, int groups, int keep, int top, float scale, float* z, int* idx, float* wts,
                             cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  if (E <= 0 || E > MOE_MAX_EXPERTS || groups <= 0 || E % groups || keep <= 0 || keep > groups || top <= 0 ||
      top > keep * (E / groups))
    return AB_BAD_ARG;
  const int wpb = 4;
  const long long lw = (long long)n_tokens * E;
  const unsigned lblocks = (unsigned)((lw + 7) / 8);
  if (dtype == AB_F32)
    ab_launch(moe_logits_kernel<float>, dim3(lblocks), dim3(256), 0, stream, (const float*)h, ld, wr, n_tokens, width, E, z, bias);
  else if (dtype == AB_BF16)
    ab_launch(moe_logits_kernel<bf16>, dim3(lblocks), dim3(256), 0, stream, (const bf16*)h, ld, wr, n_tokens, width, E, z, bias);
  else
    return AB_BAD_ARG;
  int rc = ab_launch_status();
  if (rc) return rc;
  const unsigned blocks = (unsigned)((n_tokens + wpb - 1) / wpb);
  const size_t smem = (size_t)wpb * (E + groups) * sizeof(float);
  ab_launch(moe_route_kernel, dim3(blocks), dim3(wpb * 32), smem, stream, (const float*)z, n_tokens, E, groups, keep, top,
            scale, idx, wts);
  return ab_launch_status();
}

AB_API int ab_moe_route(const void* h, int dtype, int ld, const float* wr, int n_tokens, int width, int E, int groups,
                        int keep, int top, float scale, float* z, int* idx, float* wts, cudaStream_t stream) {
  return ab_moe_route_bias(h, dtype, ld, wr, nullptr, n_tokens, width, E, groups, keep, top, scale, z, idx, wts, stream);
}

// The choice from scores that are not a softmax, one warp per token, from the logits z [T, E]:
//   s = sigmoid(z) (score_fn 1) or z itself (0);  the CHOICE is made by c = s + correction (if given), the weights
//   are the chosen experts' s, times `scale`, divided by their sum if `renorm`.
//   Groups: a group's score is the sum of its `group_top` largest c; experts outside the `keep` best groups cannot be
//   chosen whatever their c (choice scores may be negative, so they are struck out with minus infinity).
// The lower index wins a tie, among groups and among experts.
// (one token, by one warp: z its logits, s, c, gs scratch of E, E and `groups` numbers, idx and wts its `top` choices)
__device__ __forceinline__ void choose_by_scores(const float* z, const float* __restrict__ correction, int E, int groups, int keep,
                                                 int group_top, int top, int score_fn, int renorm, float scale, float* s, float* c,
                                                 float* gs, int* __restrict__ idx, float* __restrict__ wts, int lane) {
  for (int e = lane; e < E; e += 32) {
    const float v = z[e];
    const float sc = score_fn == 1 ? 1.0f / (1.0f + expf(-v)) : v;
    s[e] = sc;
    c[e] = sc + (correction != nullptr ? correction[e] : 0.f);
  }
  __syncwarp();
  const int per = E / groups;
  if (keep < groups) {
    for (int g = lane; g < groups; g += 32) {
      // the sum of the group's `group_top` largest choice scores, by repeated arg-max over a few members
      float total = 0.f;
      unsigned long long taken_lo = 0, taken_hi = 0;      // members already counted (a group of up to 128)
      for (int pick = 0; pick < group_top && pick < per; ++pick) {
        float best = -INFINITY;
        int bj = -1;
        for (int j = 0; j < per; ++j) {
          const bool used = j < 64 ? (taken_lo >> j) & 1ull : (taken_hi >> (j - 64)) & 1ull;
          if (!used && (bj < 0 || c[g * per + j] > best)) { best = c[g * per + j]; bj = j; }
        }
        if (bj < 64) taken_lo |= 1ull << bj; else taken_hi |= 1ull << (bj - 64);
        total += best;
      }
      gs[g] = total;
    }
    __syncwarp();
    for (int pick = 0; pick < keep; ++pick) {
      float best = -INFINITY;
      int bg = 0x7fffffff;
      for (int g = lane; g < groups; g += 32)
        if (!isnan(gs[g]) && (bg == 0x7fffffff || gs[g] > best)) { best = gs[g]; bg = g; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, best, o);
        const int og = __shfl_xor_sync(0xffffffffu, bg, o);
        if (og != 0x7fffffff && (bg == 0x7fffffff || ob > best || (ob == best && og < bg))) { best = ob; bg = og; }
      }
      if (lane == 0 && bg != 0x7fffffff) gs[bg] = __int_as_float(0x7fc00000);      // kept: marked with a NaN
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (!isnan(gs[e / per])) c[e] = -INFINITY;
    __syncwarp();
  }
  float chosen_sum = 0.f;
  for (int pick = 0; pick < top; ++pick) {
    float best = -INFINITY;
    int be = 0x7fffffff;
    for (int e = lane; e < E; e += 32) {
      const float v = c[e];
      if (v > best) { best = v; be = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ob > best || (ob == best && oe < be)) { best = ob; be = oe; }
    }
    if (be == 0x7fffffff) be = 0;                      // nothing left to choose (or the row holds no numbers)
    const float w = s[be];
    chosen_sum += w;
    if (lane == 0) {
      idx[pick] = be;
      wts[pick] = w;
    }
    __syncwarp();
    if (lane == 0) c[be] = -INFINITY;                  // taken
    __syncwarp();
  }
  if (lane == 0) {
    const float f = renorm ? scale / (chosen_sum + 1e-20f) : scale;
    for (int j = 0; j < top; ++j) wts[j] *= f;
  }
}

__global__ void moe_route_scores_kernel(const float* __restrict__ z, const float* __restrict__ correction, int n_tokens,
                                        int E, int groups, int keep, int group_top, int top, int score_fn, int renorm,
                                        float scale, int* __restrict__ idx, float* __restrict__ wts) {
  extern __shared__ float sm[];           // per warp: E scores, E choice scores, `groups` group scores
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31, wib = threadIdx.x >> 5;
  const int t = blockIdx.x * (blockDim.x >> 5) + wib;
  if (t >= n_tokens) return;
  float* s = sm + (size_t)wib * (2 * E + groups);
  choose_by_scores(z + (size_t)t * E, correction, E, groups, keep, group_top, top, score_fn, renorm, scale, s, s + E, s + 2 * E,
                   idx + (size_t)t * top, wts + (size_t)t * top, lane);
}

// Logits and choice of a few tokens in one kernel: a block per token, a warp per expert in turn; the router's rows are asked
// of the L2 before the wait.
template <typename T, typename TW>
__global__ void __launch_bounds__(512)
moe_route_small_kernel(const T* __restrict__ h, int ld, const TW* __restrict__ wr, const float* __restrict__ bias,
                       const float* __restrict__ correction, int width, int E, int groups, int keep, int group_top, int top,
                       int score_fn, int renorm, float scale, int* __restrict__ idx, float* __restrict__ wts) {
  extern __shared__ float sm[];           // E logits, E scores, E choice scores, `groups` group scores
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x;
  const char* rows = reinterpret_cast<const char*>(wr);
  for (size_t at = (size_t)threadIdx.x * 128; at < (size_t)E * width * sizeof(TW); at += (size_t)blockDim.x * 128)
    asm volatile("prefetch.global.L2 [%0];" ::"l"(rows + at));
  pdl_wait();
  pdl_trigger();
  for (int e = warp; e < E; e += blockDim.x >> 5) {
    const float part = warp_sum(lane_dot(h + (size_t)t * ld, wr + (size_t)e * width, width, lane));
    if (lane == 0) sm[e] = part + (bias != nullptr ? bias[e] : 0.f);
  }
  __syncthreads();
  if (warp == 0)
    choose_by_scores(sm, correction, E, groups, keep, group_top, top, score_fn, renorm, scale, sm + E, sm + 2 * E, sm + 3 * E,
                     idx + (size_t)t * top, wts + (size_t)t * top, lane);
}

static bool route_ok(int E, int groups, int keep, int group_top, int top, int score_fn) {
  return E > 0 && E <= MOE_MAX_EXPERTS && groups > 0 && E % groups == 0 && keep > 0 && keep <= groups && top > 0 &&
         top <= keep * (E / groups) && group_top > 0 && !(keep < groups && E / groups > 128) && score_fn >= 0 && score_fn <= 1;
}

// The choice of every token from its logits z [T, E].
AB_API int ab_moe_route_logits(const float* z, const float* correction, int n_tokens, int E, int groups, int keep, int group_top,
                               int top, int score_fn, int renorm, float scale, int* idx, float* wts, cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  if (!route_ok(E, groups, keep, group_top, top, score_fn)) return AB_BAD_ARG;
  const int wpb = 4;
  const unsigned blocks = (unsigned)((n_tokens + wpb - 1) / wpb);
  const size_t smem = (size_t)wpb * (2 * E + groups) * sizeof(float);
  ab_launch(moe_route_scores_kernel, dim3(blocks), dim3(wpb * 32), smem, stream, z, correction, n_tokens, E, groups, keep, group_top,
            top, score_fn, renorm, scale, idx, wts);
  return ab_launch_status();
}

AB_API int ab_moe_route_scores(const void* h, int dtype, int ld, const float* wr, const float* bias, const float* correction,
                               int n_tokens, int width, int E, int groups, int keep, int group_top, int top, int score_fn,
                               int renorm, float scale, float* z, int* idx, float* wts, cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  if (!route_ok(E, groups, keep, group_top, top, score_fn)) return AB_BAD_ARG;
  const long long lw = (long long)n_tokens * E;
  const unsigned lblocks = (unsigned)((lw + 7) / 8);
  if (dtype == AB_F32)
    ab_launch(moe_logits_kernel<float>, dim3(lblocks), dim3(256), 0, stream, (const float*)h, ld, wr, n_tokens, width, E, z, bias);
  else if (dtype == AB_BF16)
    ab_launch(moe_logits_kernel<bf16>, dim3(lblocks), dim3(256), 0, stream, (const bf16*)h, ld, wr, n_tokens, width, E, z, bias);
  else
    return AB_BAD_ARG;
  int rc = ab_launch_status();
  if (rc) return rc;
  return ab_moe_route_logits(z, correction, n_tokens, E, groups, keep, group_top, top, score_fn, renorm, scale, idx, wts, stream);
}

// Both in one kernel, for a few tokens; wr of wr_dtype (bfloat16 with bfloat16 rows of h only).
AB_API int ab_moe_route_small(const void* h, int dtype, int ld, const void* wr, int wr_dtype, const float* bias,
                              const float* correction, int n_tokens, int width, int E, int groups, int keep, int group_top, int top,
                              int score_fn, int renorm, float scale, int* idx, float* wts, cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  if (!route_ok(E, groups, keep, group_top, top, score_fn) || width <= 0) return AB_BAD_ARG;
  const size_t smem = (size_t)(3 * E + groups) * sizeof(float);
#define AB_GO(T, TW)                                                                                                   \
  ab_launch(moe_route_small_kernel<T, TW>, dim3((unsigned)n_tokens), dim3(512), smem, stream, (const T*)h, ld, (const TW*)wr, bias, \
            correction, width, E, groups, keep, group_top, top, score_fn, renorm, scale, idx, wts)
  if (dtype == AB_F32 && wr_dtype == AB_F32) AB_GO(float, float);
  else if (dtype == AB_BF16 && wr_dtype == AB_F32) AB_GO(bf16, float);
  else if (dtype == AB_BF16 && wr_dtype == AB_BF16) AB_GO(bf16, bf16);
  else return AB_BAD_ARG;
#undef AB_GO
  return ab_launch_status();
}

// act[p, j] = f(W_up[e_p][j] . h[t_p]) for pair p = t * top + k, or, gated (w_gate given),
// f(W_gate[e_p][j] . h[t_p]) * (W_up[e_p][j] . h[t_p]).  One warp per (pair, j).
template <typename T>
__global__ void moe_up_pairs_kernel(const T* __restrict__ h, int ld, const T* __restrict__ w_up, const T* __restrict__ w_gate,
                                    const int* __restrict__ idx, T* __restrict__ act, int n_pairs, int top, int width,
                                    int ff, int activation) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const long long id = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (id >= (long long)n_pairs * ff) return;
  const int p = (int)(id / ff), j = (int)(id - (long long)p * ff);
  const int e = idx[p];
  const T* x = h + (size_t)(p / top) * ld;
  const float part = warp_sum(lane_dot(x, w_up + ((size_t)e * ff + j) * width, width, lane));
  if (w_gate != nullptr) {
    const float gate = warp_sum(lane_dot(x, w_gate + ((size_t)e * ff + j) * width, width, lane));
    if (lane == 0) act[(size_t)p * ff + j] = from_f32<T>((activation == 0 ? gelu_erf(gate) : silu(gate)) * part);
    return;
  }
  if (lane == 0) {
    act[(size_t)p * ff + j] = from_f32<T>(activation == 0 ? gelu_erf(part) : silu(part));
  }
}

// out[t, i] = sum_k wts[t, k] * (W_down[e_k][i] . act[t * top + k]).  One warp per (token, i).
// w_down: [width, E, ff], the experts side by side in a row (the layout of one product over all experts).
template <typename T>
__global__ void moe_down_pairs_kernel(const T* __restrict__ act, const T* __restrict__ w_down, const int* __restrict__ idx,
                                      const float* __restrict__ wts, T* __restrict__ out, int n_tokens, int top, int width,
                                      int ff, int E) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const long long id = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (id >= (long long)n_tokens * width) return;
  const int t = (int)(id / width), i = (int)(id - (long long)t * width);
  // a lane adds up its share of all chosen experts' rows, weighted; one sum over the warp at the end, so that the
  // rows of different experts are asked for together
  float total = 0.f;
#pragma unroll 4
  for (int k = 0; k < top; ++k) {
    const int e = idx[(size_t)t * top + k];
    const float part = lane_dot(act + ((size_t)t * top + k) * ff, w_down + ((size_t)i * E + e) * ff, ff, lane);
    total = fmaf(wts[(size_t)t * top + k], part, total);
  }
  total = warp_sum(total);
  if (lane == 0) out[(size_t)t * width + i] = from_f32<T>(total);
}

// `w_gate`: [E, ff, width] for gated experts, or null
AB_API int ab_moe_pairs_gated(const void* h, int dtype, int ld, const void* w_up, const void* w_gate, const void* w_down,
                              const int* idx, const float* wts, void* act, void* out, int n_tokens, int top, int width,
                              int ff, int E, int activation, cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  if (top <= 0 || width <= 0 || ff <= 0 || E <= 0 || (activation != 0 && activation != 1)) return AB_BAD_ARG;
  const int wpb = 8;
  const long long up_warps = (long long)n_tokens * top * ff, down_warps = (long long)n_tokens * width;
  const long long up_blocks = (up_warps + wpb - 1) / wpb, down_blocks = (down_warps + wpb - 1) / wpb;
  if (up_blocks > 0x7fffffffLL || down_blocks > 0x7fffffffLL) return AB_BAD_ARG;
  if (dtype == AB_F32) {
    ab_launch(moe_up_pairs_kernel<float>, dim3((unsigned)up_blocks), dim3(wpb * 32), 0, stream, (const float*)h, ld,
              (const float*)w_up, (const float*)w_gate, idx, (float*)act, n_tokens * top, top, width, ff, activation);
    ab_launch(moe_down_pairs_kernel<float>, dim3((unsigned)down_blocks), dim3(wpb * 32), 0, stream, (const float*)act,
              (const float*)w_down, idx, wts, (float*)out, n_tokens, top, width, ff, E);
  } else if (dtype == AB_BF16) {
    ab_launch(moe_up_pairs_kernel<bf16>, dim3((unsigned)up_blocks), dim3(wpb * 32), 0, stream, (const bf16*)h, ld,
              (const bf16*)w_up, (const bf16*)w_gate, idx, (bf16*)act, n_tokens * top, top, width, ff, activation);
    ab_launch(moe_down_pairs_kernel<bf16>, dim3((unsigned)down_blocks), dim3(wpb * 32), 0, stream, (const bf16*)act,
              (const bf16*)w_down, idx, wts, (bf16*)out, n_tokens, top, width, ff, E);
  } else {
    return AB_BAD_ARG;
  }
  return ab_launch_status();
}

AB_API int ab_moe_pairs(const void* h, int dtype, int ld, const void* w_up, const void* w_down, const int* idx,
                        const float* wts, void* act, void* out, int n_tokens, int top, int width, int ff, int E,
                        int activation, cudaStream_t stream) {
  return ab_moe_pairs_gated(h, dtype, ld, w_up, nullptr, w_down, idx, wts, act, out, n_tokens, top, width, ff, E,
                            activation, stream);
}

// All experts at once, for steps of many tokens: up[t, e * ff + j] holds W_up[e][j] . h[t] for every expert
// (one product); in place it becomes act(up) * (the token's weight for expert e, 0 if e was not chosen), so
// that one product with the experts side by side, [width, E * ff], adds the chosen experts' outputs.
// Gated: a row of `up` holds the gates of all experts and then their up-projections (2 * E * ff numbers); the result
// takes the gates' place.
template <typename T>
__global__ void moe_weigh_all_kernel(T* __restrict__ up, const int* __restrict__ idx, const float* __restrict__ wts,
                                     int n_tokens, int top, int ff, int E, int activation, int gated) {
  const int t = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;       // column in [0, E * ff)
  if (c >= E * ff) return;
  const int e = c / ff;
  float g = 0.f;
  for (int k = 0; k < top; ++k)
    if (idx[(size_t)t * top + k] == e) g = wts[(size_t)t * top + k];
  T* x = up + (size_t)t * E * ff * (gated ? 2 : 1) + c;
  float y = 0.f;
  if (g != 0.f) {
    const float z = to_f32(*x);
    y = g * (activation == 0 ? gelu_erf(z) : silu(z));
    if (gated) y *= to_f32(x[(size_t)E * ff]);
  }
  *x = from_f32<T>(y);
}

// the same, eight bfloat16 columns per thread (ff a multiple of 8: the eight belong to one expert); the columns
// of experts that were not chosen are written without being read
__global__ void moe_weigh_all_bf16x8_kernel(bf16* __restrict__ up, const int* __restrict__ idx,
                                            const float* __restrict__ wts, int n_tokens, int top, int ff, int E,
                                            int activation, int gated) {
  const int t = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= E * ff) return;
  const int e = c / ff;
  float g = 0.f;
  for (int k = 0; k < top; ++k)
    if (idx[(size_t)t * top + k] == e) g = wts[(size_t)t * top + k];
  uint4* x = reinterpret_cast<uint4*>(up + (size_t)t * E * ff * (gated ? 2 : 1) + c);
  uint4 v = make_uint4(0, 0, 0, 0);
  if (g != 0.f) {
    v = *x;
    uint4 u = make_uint4(0, 0, 0, 0);
    if (gated) u = *reinterpret_cast<const uint4*>(up + (size_t)t * E * ff * 2 + (size_t)E * ff + c);
    __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&v);
    const __nv_bfloat162* pu = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float2 z = __bfloat1622float2(p[j]);
      z.x = g * (activation == 0 ? gelu_erf(z.x) : silu(z.x));
      z.y = g * (activation == 0 ? gelu_erf(z.y) : silu(z.y));
      if (gated) {
        const float2 m = __bfloat1622float2(pu[j]);
        z.x *= m.x;
        z.y *= m.y;
      }
      p[j] = __floats2bfloat162_rn(z.x, z.y);
    }
  }
  *x = v;
}

AB_API int ab_moe_weigh_all_gated(void* up, int dtype, const int* idx, const float* wts, int n_tokens, int top, int ff,
                                  int E, int activation, int gated, cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  if (top <= 0 || ff <= 0 || E <= 0 || n_tokens > 65535 || (activation != 0 && activation != 1)) return AB_BAD_ARG;
  dim3 grid((unsigned)(((long long)E * ff + 255) / 256), (unsigned)n_tokens);
  if (dtype == AB_F32)
    moe_weigh_all_kernel<float><<<grid, 256, 0, stream>>>((float*)up, idx, wts, n_tokens, top, ff, E, activation, gated);
  else if (dtype == AB_BF16 && ff % 8 == 0 && (((uintptr_t)up) & 15) == 0) {
    dim3 grid8((unsigned)(((long long)E * ff / 8 + 255) / 256), (unsigned)n_tokens);
    moe_weigh_all_bf16x8_kernel<<<grid8, 256, 0, stream>>>((bf16*)up, idx, wts, n_tokens, top, ff, E, activation, gated);
  } else if (dtype == AB_BF16)
    moe_weigh_all_kernel<bf16><<<grid, 256, 0, stream>>>((bf16*)up, idx, wts, n_tokens, top, ff, E, activation, gated);
  else
    return AB_BAD_ARG;
  return ab_launch_status();
}

AB_API int ab_moe_weigh_all(void* up, int dtype, const int* idx, const float* wts, int n_tokens, int top, int ff, int E,
                            int activation, cudaStream_t stream) {
  return ab_moe_weigh_all_gated(up, dtype, idx, wts, n_tokens, top, ff, E, activation, 0, stream);
}

// ---------------------------------------------------------------------------
// Experts behind any choice, with a shared expert.
//
//   y_t = sum_k weight_k W_down[e_k] (silu(W_gate[e_k] h_t) * (W_up[e_k] h_t))
//         + sigmoid(z_t) W_down_s (silu(W_gate_s h_t) * (W_up_s h_t))               (if there is a shared expert)
//
// without gates: W_down[e_k] act(W_up[e_k] h_t), gate_up then holds the up-projections alone, [E * ff, width].  With
// `weight_in` weight_k multiplies expert k's input instead of its output.  z null: the shared expert's factor is 1.
//
// The choice comes from a router (`idx`, `wts`) or from the token's id: a row of a table names its experts, each with the
// same constant weight (moe_choice.cuh).  Layouts (ff and fs multiples of 8): gate_up [E, 2 ff, width], an expert's rows in
// groups of 16, the gates of 8 units and then their up-projections; down [E, width, ff]; the shared expert's likewise,
// [2 fs, width] and [width, fs].  z [T] are the shared expert's gate logits (float32, formed elsewhere).
// The pair kernels here take any width and the 32-bit path.  bfloat16 steps of a few tokens run csrc/moe_gemv.cu; steps of
// many tokens sort their (token, expert) pairs by expert (moe_plan), copy the tokens' rows into that order (moe_gather),
// run two grouped products (csrc/gemm_tc.cu) and add up each token's outputs (moe_combine).
// ---------------------------------------------------------------------------
__device__ __forceinline__ void fma8(float& part, uint4 x, uint4 y) {
  const uint32_t a[4] = {x.x, x.y, x.z, x.w}, b[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    part = fmaf(__uint_as_float(a[j] << 16), __uint_as_float(b[j] << 16), part);
    part = fmaf(__uint_as_float(a[j] & 0xffff0000u), __uint_as_float(b[j] & 0xffff0000u), part);
  }
}
// A warp's shares of x . g and x . u (rows of n numbers): the rows' 16-byte pieces are asked for four at a time each.
__device__ __forceinline__ void lane_dot2(const bf16* __restrict__ x, const bf16* __restrict__ g, const bf16* __restrict__ u,
                                          int n, int lane, float& pg, float& pu) {
  pg = pu = 0.f;
  if ((n & 7) == 0 && ((((uintptr_t)x) | ((uintptr_t)g) | ((uintptr_t)u)) & 15) == 0) {
    for (int k0 = lane * 8; k0 < n; k0 += 1024) {
      uint4 gv[4], uv[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int k = k0 + j * 256;
        gv[j] = uv[j] = make_uint4(0, 0, 0, 0);
        if (k < n) {
          gv[j] = __ldg(reinterpret_cast<const uint4*>(g + k));
          uv[j] = __ldg(reinterpret_cast<const uint4*>(u + k));
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int k = k0 + j * 256;
        if (k < n) {
          const uint4 xv = *reinterpret_cast<const uint4*>(x + k);
          fma8(pg, xv, gv[j]);
          fma8(pu, xv, uv[j]);
        }
      }
    }
    return;
  }
  for (int k = lane; k < n; k += 32) {
    const float v = __bfloat162float(x[k]);
    pg = fmaf(v, __bfloat162float(g[k]), pg);
    pu = fmaf(v, __bfloat162float(u[k]), pu);
  }
}
__device__ __forceinline__ void lane_dot2(const float* __restrict__ x, const float* __restrict__ g, const float* __restrict__ u,
                                          int n, int lane, float& pg, float& pu) {
  pg = pu = 0.f;
  for (int k = lane; k < n; k += 32) {
    pg = fmaf(x[k], g[k], pg);
    pu = fmaf(x[k], u[k], pu);
  }
}

// act: [T, top * ff + fs].  A block of eight warps takes one unit of an expert for eight (token, choice) pairs, or one
// unit of the shared expert for eight tokens, whose warps then read the same two rows at the same time.
template <typename T, bool GATED>
__global__ void __launch_bounds__(256)
moe_shared_up_kernel(const T* __restrict__ h, int ld, const T* __restrict__ gate_up, const T* __restrict__ gate_up_s, Choice c,
                     T* __restrict__ act, int n_tokens, int top, int width, int ff, int fs, int E, int activation, int weight_in,
                     long long pair_blocks) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_wait();
  pdl_trigger();
  const int row_len = top * ff + fs;
  int t;
  float wgt = 1.0f;
  size_t unit, dst;
  const T* w = gate_up;
  long long blk = blockIdx.x;
  if (blk < pair_blocks) {
    const long long group = blk / ff;
    const int j = (int)(blk - group * ff);
    const long long p = group * 8 + warp;
    if (p >= (long long)n_tokens * top) return;
    t = (int)(p / top);
    const int k = (int)(p - (long long)t * top);
    unit = (size_t)chosen_expert(c, t, k, top) * ff + j;
    dst = (size_t)t * row_len + (size_t)k * ff + j;
    if (weight_in) wgt = chosen_weight(c, t, k, top);
  } else {
    blk -= pair_blocks;
    const int chunk = (int)(blk / fs), j = (int)(blk - (long long)chunk * fs);
    t = chunk * 8 + warp;
    if (t >= n_tokens) return;
    unit = j;
    w = gate_up_s;
    dst = (size_t)t * row_len + (size_t)top * ff + j;
  }
  float pg = 0.f, pu;
  if (GATED) {
    const T* gate = w + ((unit >> 3) * 16 + (unit & 7)) * width;
    lane_dot2(h + (size_t)t * ld, gate, gate + (size_t)8 * width, width, lane, pg, pu);
    pg = warp_sum(pg);
  } else {
    pu = lane_dot(h + (size_t)t * ld, w + unit * width, width, lane);
  }
  pu = warp_sum(pu);
  // (a weight on the output is applied by the down-projection)
  if (lane == 0) act[dst] = from_f32<T>(expert_inner<GATED>(pg, pu, wgt, 1, activation));
}

// out[t, i], float32 or T.  A block of eight warps takes one column i for eight tokens (the shared expert's row is then
// read by all of them together).
template <typename T, typename TO>
__global__ void __launch_bounds__(256)
moe_shared_down_kernel(const T* __restrict__ act, const T* __restrict__ down, const T* __restrict__ down_s, Choice c,
                       const float* __restrict__ z, TO* __restrict__ out, int n_tokens, int top, int width, int ff, int fs, int E,
                       int weight_in) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_wait();
  pdl_trigger();
  const int i = blockIdx.x, t = blockIdx.y * 8 + warp;
  if (t >= n_tokens) return;
  const T* a = act + (size_t)t * (top * ff + fs);
  float total = 0.f;
#pragma unroll 4
  for (int k = 0; k < top; ++k) {
    const int e = chosen_expert(c, t, k, top);
    const float part = lane_dot(a + (size_t)k * ff, down + ((size_t)e * width + i) * ff, ff, lane);
    total = fmaf(weight_in ? 1.0f : chosen_weight(c, t, k, top), part, total);
  }
  if (fs > 0) {
    const float part = lane_dot(a + (size_t)top * ff, down_s + (size_t)i * fs, fs, lane);
    total = fmaf(z != nullptr ? 1.0f / (1.0f + expf(-z[t])) : 1.0f, part, total);
  }
  total = warp_sum(total);
  if (lane == 0) out[(size_t)t * width + i] = from_f32<TO>(total);
}

// act: scratch [n_tokens, top * ff + fs] of `dtype`; out of `out_dtype`.
AB_API int ab_moe_shared_pairs(const void* h, int dtype, int ld, const void* gate_up, const void* down, const void* gate_up_s,
                               const void* down_s, const int* idx, const float* wts, const int* table, const int* tokens, float weight, const float* z, void* act,
                               void* out, int out_dtype, int n_tokens, int top, int width, int ff, int fs, int E,
                               int activation, int gated, int weight_in, cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  const Choice c{idx, wts, table, tokens, weight};
  if (top <= 0 || width <= 0 || ff <= 0 || ff % 8 || fs < 0 || fs % 8 || E <= 0 || activation < 0 || activation >= MOE_ACT_KINDS ||
      !choice_ok(c) || (fs > 0 && (!gate_up_s || !down_s)))
    return AB_BAD_ARG;
  const long long pair_blocks = ((long long)n_tokens * top + 7) / 8 * ff;
  const long long blocks = pair_blocks + ((long long)n_tokens + 7) / 8 * fs;
  if (blocks > 0x7fffffffLL || width > 0x7fffffff || (n_tokens + 7) / 8 > 65535) return AB_BAD_ARG;
  const dim3 dgrid((unsigned)width, (unsigned)((n_tokens + 7) / 8));
#define AB_GO(T, TO)                                                                                                   \
  {                                                                                                                    \
    ab_launch(gated ? moe_shared_up_kernel<T, true> : moe_shared_up_kernel<T, false>, dim3((unsigned)blocks), dim3(256), 0, \
              stream, (const T*)h, ld, (const T*)gate_up, (const T*)gate_up_s, c, (T*)act, n_tokens, top, width, ff, fs, E, \
              activation, weight_in, pair_blocks);                                                                     \
    ab_launch(moe_shared_down_kernel<T, TO>, dgrid, dim3(256), 0, stream, (const T*)act, (const T*)down, (const T*)down_s, c, z, (TO*)out, \
              n_tokens, top, width, ff, fs, E, weight_in);                                                             \
  }
  if (dtype == AB_F32 && out_dtype == AB_F32) AB_GO(float, float)
  else if (dtype == AB_BF16 && out_dtype == AB_F32) AB_GO(bf16, float)
  else if (dtype == AB_BF16 && out_dtype == AB_BF16) AB_GO(bf16, bf16)
  else return AB_BAD_ARG;
#undef AB_GO
  return ab_launch_status();
}

// ---------------------------------------------------------------------------
// many tokens: the pairs in order of their experts
// ---------------------------------------------------------------------------
#define MOE_TILE 128           // rows of a row tile of the grouped product

// pos[t * top + k]: the row of a pair; an expert's rows start on a row tile.  tile_group[i]: the expert of row tile i,
// row_tiles[0]: how many row tiles there are.  row_weight (or null): a pair's weight, by its row.  One block; the order of an expert's rows among themselves is whatever the
// counters give (a row's result does not depend on its place).
__global__ void __launch_bounds__(1024)
moe_plan_kernel(Choice c, int n_tokens, int top, int E, int* __restrict__ pos, int* __restrict__ tile_group,
                int* __restrict__ row_tiles, float* __restrict__ row_weight) {
  __shared__ int count[MOE_MAX_EXPERTS], first[MOE_MAX_EXPERTS];
  pdl_wait();
  pdl_trigger();
  for (int e = threadIdx.x; e < E; e += blockDim.x) count[e] = 0;
  __syncthreads();
  // eight pairs per thread at a time, their loads together; the first eight stay in registers for the second pass
  const int n_pairs = n_tokens * top;
  int mine[8];
  for (int p0 = threadIdx.x; p0 < n_pairs; p0 += 8 * blockDim.x) {
    int e[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int p = p0 + j * blockDim.x;
      e[j] = p < n_pairs ? chosen_expert(c, p / top, p % top, top) : -1;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (e[j] >= 0) atomicAdd(&count[e[j]], 1);
      if (p0 == (int)threadIdx.x) mine[j] = e[j];
    }
  }
  __syncthreads();
  if (threadIdx.x < 32) {                      // the experts' first row tiles: a running sum over lanes
    int before = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const int tiles = e < E ? (count[e] + MOE_TILE - 1) / MOE_TILE : 0;
      int incl = tiles;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, incl, o);
        if ((int)threadIdx.x >= o) incl += up;
      }
      if (e < E) {
        first[e] = (before + incl - tiles) * MOE_TILE;
        for (int i = 0; i < tiles; ++i) tile_group[before + incl - tiles + i] = e;
      }
      before += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (threadIdx.x == 0) *row_tiles = before;
  }
  __syncthreads();
  for (int p0 = threadIdx.x; p0 < n_pairs; p0 += 8 * blockDim.x) {
    int e[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int p = p0 + j * blockDim.x;
      e[j] = p0 == (int)threadIdx.x ? mine[j] : p < n_pairs ? chosen_expert(c, p / top, p % top, top) : -1;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (e[j] >= 0) {
        const int p = p0 + j * blockDim.x, row = atomicAdd(&first[e[j]], 1);
        pos[p] = row;
        if (row_weight != nullptr) row_weight[row] = chosen_weight(c, p / top, p % top, top);
      }
  }
}

// rows[pos[t, k]] = h[t] for every choice k; 16-byte pieces (width a multiple of 8)
__global__ void __launch_bounds__(256)
moe_gather_kernel(const bf16* __restrict__ h, const int* __restrict__ pos, bf16* __restrict__ rows, int top, int width) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  for (int i = threadIdx.x * 8; i < width; i += blockDim.x * 8) {
    const uint4 v = *reinterpret_cast<const uint4*>(h + (size_t)t * width + i);
    for (int k = 0; k < top; ++k)
      *reinterpret_cast<uint4*>(rows + (size_t)pos[(size_t)t * top + k] * width + i) = v;
  }
}

// out[t] = sum_k weight_k y[pos[t, k]] + sigmoid(z_t) ys[t]   (ys null: no shared expert; z null: its factor is 1;
// `weighed`: the rows of y carry their weights already)
__global__ void __launch_bounds__(256)
moe_combine_kernel(const bf16* __restrict__ y, const int* __restrict__ pos, Choice c, const bf16* __restrict__ ys,
                   const float* __restrict__ z, float* __restrict__ out, int top, int width, int weighed) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  const float g = z != nullptr ? 1.0f / (1.0f + expf(-z[t])) : 1.0f;
  for (int i = threadIdx.x * 8; i < width; i += blockDim.x * 8) {
    float s[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) s[j] = 0.f;
    auto add = [&](const bf16* p, float w) {
      const uint4 v = *reinterpret_cast<const uint4*>(p);
      const uint32_t a[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        s[2 * j] = fmaf(w, __uint_as_float(a[j] << 16), s[2 * j]);
        s[2 * j + 1] = fmaf(w, __uint_as_float(a[j] & 0xffff0000u), s[2 * j + 1]);
      }
    };
#pragma unroll 4
    for (int k = 0; k < top; ++k) add(y + (size_t)pos[(size_t)t * top + k] * width + i, weighed ? 1.0f : chosen_weight(c, t, k, top));
    if (ys != nullptr) add(ys + (size_t)t * width + i, g);
    float4* o = reinterpret_cast<float4*>(out + (size_t)t * width + i);
    o[0] = make_float4(s[0], s[1], s[2], s[3]);
    o[1] = make_float4(s[4], s[5], s[6], s[7]);
  }
}

// pos int [n_tokens * top], tile_group int [n_tokens * top / 128 + E], row_tiles int [1]; rows bfloat16
// [(n_tokens * top / 128 + E) * 128, width].
AB_API int ab_moe_gather(const void* h, const int* idx, const float* wts, const int* table, const int* tokens, float weight,
                         int* pos, int* tile_group, int* row_tiles, float* row_weight, void* rows, int n_tokens, int top, int width, int E,
                         cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  const Choice c{idx, wts, table, tokens, weight};
  if (top <= 0 || E <= 0 || E > MOE_MAX_EXPERTS || width <= 0 || width % 8 || !choice_ok(c) ||
      (long long)n_tokens * top > 0x3fffffffLL || ((((uintptr_t)h) | ((uintptr_t)rows)) & 15))
    return AB_BAD_ARG;
  ab_launch(moe_plan_kernel, dim3(1), dim3(1024), 0, stream, c, n_tokens, top, E, pos, tile_group, row_tiles,
            row_weight);
  ab_launch(moe_gather_kernel, dim3((unsigned)n_tokens), dim3(width >= 2048 ? 256 : 128), 0, stream, (const bf16*)h,
            (const int*)pos, (bf16*)rows, top, width);
  return ab_launch_status();
}

AB_API int ab_moe_combine(const void* y, const int* pos, const int* idx, const float* wts, const int* table, const int* tokens,
                          float weight, const void* ys, const float* z, float* out, int n_tokens, int top, int width, int weighed,
                          cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  const Choice c{idx, wts, table, tokens, weight};
  if (top <= 0 || width <= 0 || width % 8 || !choice_ok(c) ||
      ((((uintptr_t)y) | ((uintptr_t)ys) | ((uintptr_t)out)) & 15))
    return AB_BAD_ARG;
  ab_launch(moe_combine_kernel, dim3((unsigned)n_tokens), dim3(width >= 2048 ? 256 : 128), 0, stream, (const bf16*)y, pos, c,
            (const bf16*)ys, z, out, top, width, weighed);
  return ab_launch_status();
}

// Experts (gated or not) with a shared expert for bfloat16 steps of up to 32 tokens: two skinny products whose weights are read
// once from memory, for all tokens that chose an expert together.  (The kernels of moe.cu read an expert's rows once per
// (token, expert) pair: with several tokens per expert that is several times the weights' bytes through the L2.)
//
//   up    a CTA owns 8 units of one expert (16 rows of gate_up: 8 gates, 8 up-projections) or of the shared expert.  It
//         lists the tokens that chose the expert (from the choice, which is known before the kernel before this one has
//         ended), leaves if there are none, and multiplies its rows with those tokens' rows on the tensor cores
//         (mma.sync m16n8k16, the weights as the 16-row operand, the listed tokens as the columns; see gemv_bf16.cu for
//         the loads and the permutation of k).  act[t, slot, unit] = weight * act(gate) * up, the weight being the
//         choice's or, for the shared expert, sigmoid(z_t) (1 without z).  Without gates the 16 rows are 16 units,
//         weight * act(up); with `weight_in` a chosen expert's weight multiplies its input instead.
//   down  a CTA owns 16 columns of the output and walks the units of the experts that were chosen by any token, then the
//         shared expert's; a token's column is zero where it did not choose the expert.  The walk is cut into slices, the
//         CTAs of a cluster, whose sums the first of them adds in slice order.
//
// Sums are float32: a warp's over its run of units, then the warps' in order, then the slices' in order.
#include "common.cuh"
#include "launch.cuh"
#include "moe_choice.cuh"
#include <cooperative_groups.h>

#define MG_U 8                 // k-groups (32 numbers) a thread asks for before it uses any
#define MG_MAX_TOKENS 32
#define MG_MAX_EXPERTS 512
#define MG_MAX_TOP 32

__device__ __forceinline__ void mg_mma(float* c, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
               "{%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint4 mg_stream(const void* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
// activations were written by the kernel before this one: a coherent load
__device__ __forceinline__ uint4 mg_act(const bf16* p) {
  uint4 v;
  asm volatile("ld.global.v4.u32 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p) : "memory");
  return v;
}

template <int NT, bool GATED>
__global__ void __launch_bounds__(256)
moe_gemv_up_kernel(const bf16* __restrict__ X, const bf16* __restrict__ W, const bf16* __restrict__ Ws, Choice c, const float* __restrict__ z,
                   bf16* __restrict__ act, int M, int K, int top, int ff, int fs, int E, int activation,
                   int weight_in) {
  constexpr int UNITS = GATED ? 8 : 16;        // of a slab of 16 rows
  constexpr int WARPS = 8;
  __shared__ float red[WARPS][NT][32][4];
  __shared__ int list[NT * 8];                  // token * top + slot (the shared expert: token * top + top, one slot more)
  __shared__ int n_list;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, t = lane & 3;
  const int slab = blockIdx.x, per_expert = ff / UNITS;
  const bool shared = slab >= E * per_expert;
  const int e = shared ? E : slab / per_expert;
  const int unit0 = (shared ? slab - E * per_expert : slab - e * per_expert) * UNITS;      // within the expert
  bool waited = false;
  if (c.idx != nullptr) { pdl_wait(); pdl_trigger(); waited = true; }      // a router's choice is the kernel's before this one
  if (warp == 0) {
    int slot = -1;
    if (lane < M) {
      if (shared) slot = top;
      else
        for (int k = 0; k < top; ++k)
          if (chosen_expert(c, lane, k, top) == e) slot = k;
    }
    const unsigned who = __ballot_sync(0xffffffffu, slot >= 0);
    if (slot >= 0) list[__popc(who & ((1u << lane) - 1u))] = lane * (top + 1) + slot;
    if (lane == 0) n_list = __popc(who);
  }
  __syncthreads();
  const int n = n_list;
  if (n == 0) {
    if (!waited) { pdl_wait(); pdl_trigger(); }
    return;
  }
  const bf16* w_lo = (shared ? Ws + (size_t)(slab - E * per_expert) * 16 * K : W + (size_t)slab * 16 * K) + (size_t)g * K;
  const bf16* w_hi = w_lo + (size_t)8 * K;
  const bf16* x_row[NT];
  bool x_ok[NT];
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    x_ok[i] = i * 8 + g < n;
    x_row[i] = X + (size_t)(x_ok[i] ? list[i * 8 + g] / (top + 1) : 0) * K;
  }
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  const int n_groups = (K + 31) / 32;
  const int per_warp = (n_groups + WARPS - 1) / WARPS;
  const int begin = warp * per_warp, end = min(n_groups, begin + per_warp);
  for (int grp = begin; grp < end; grp += MG_U) {
    uint4 wl[MG_U], wh[MG_U];
#pragma unroll
    for (int u = 0; u < MG_U; ++u) {
      const int k = (grp + u) * 32 + t * 8;
      wl[u] = wh[u] = make_uint4(0, 0, 0, 0);
      if (grp + u < end && k < K) {
        wl[u] = mg_stream(w_lo + k);
        wh[u] = mg_stream(w_hi + k);
      }
    }
    if (!waited) { pdl_wait(); pdl_trigger(); waited = true; }
#pragma unroll
    for (int u0 = 0; u0 < MG_U; u0 += 4) {
      uint4 xv[4][NT];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int k = (grp + u0 + u) * 32 + t * 8;
        const bool in = grp + u0 + u < end && k < K;
#pragma unroll
        for (int i = 0; i < NT; ++i) xv[u][i] = (in && x_ok[i]) ? mg_act(x_row[i] + k) : make_uint4(0, 0, 0, 0);
      }
#pragma unroll
      for (int u = 0; u < 4; ++u)
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          mg_mma(acc[i], wl[u0 + u].x, wh[u0 + u].x, wl[u0 + u].y, wh[u0 + u].y, xv[u][i].x, xv[u][i].y);
          mg_mma(acc[i], wl[u0 + u].z, wh[u0 + u].z, wl[u0 + u].w, wh[u0 + u].w, xv[u][i].z, xv[u][i].w);
        }
    }
  }
  if (!waited) { pdl_wait(); pdl_trigger(); }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) red[warp][i][lane][j] = acc[i][j];
  __syncthreads();
  if (threadIdx.x >= NT * 32) return;
  const int i = threadIdx.x >> 5;
  float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int w = 0; w < WARPS; ++w)
#pragma unroll
    for (int j = 0; j < 4; ++j) s[j] += red[w][i][lane][j];
  const int row_len = top * ff + fs;
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int at = i * 8 + 2 * t + j;          // columns 2t, 2t + 1: listed tokens; s[j], s[2 + j]: rows g and g + 8
    if (at >= n) continue;
    const int tok = list[at] / (top + 1), slot = list[at] - tok * (top + 1);
    const float wgt = !shared ? chosen_weight(c, tok, slot, top) : z != nullptr ? 1.0f / (1.0f + expf(-z[tok])) : 1.0f;
    const int in = shared ? 0 : weight_in;
    bf16* dst = act + (size_t)tok * row_len + (size_t)slot * ff + unit0 + g;
    if (GATED) {
      *dst = __float2bfloat16_rn(expert_inner<true>(s[j], s[2 + j], wgt, in, activation));
    } else {
      dst[0] = __float2bfloat16_rn(expert_inner<false>(0.f, s[j], wgt, in, activation));
      dst[8] = __float2bfloat16_rn(expert_inner<false>(0.f, s[2 + j], wgt, in, activation));
    }
  }
}

template <int NT, int WARPS>
__global__ void __launch_bounds__(WARPS * 32)
moe_gemv_down_kernel(const bf16* __restrict__ act, const bf16* __restrict__ W, const bf16* __restrict__ Ws, Choice c, float* __restrict__ out, int M, int N,
                     int top, int ff, int fs, int E, int slices) {
  namespace cg = cooperative_groups;
  __shared__ float red[WARPS][NT][32][4];
  __shared__ float tile[NT][32][4];                          // this slice's sums, read by the cluster's first CTA
  __shared__ signed char slot_of[MG_MAX_EXPERTS][NT * 8];    // a token's slot of an expert, -1: not chosen
  __shared__ short active[MG_MAX_EXPERTS];
  __shared__ bool picked[MG_MAX_EXPERTS];
  __shared__ int n_active;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3;
  const int n0 = blockIdx.x * 16, slice = blockIdx.y;
  __shared__ short chosen[MG_MAX_TOKENS * MG_MAX_TOP];
  for (int i = tid; i < M * top; i += WARPS * 32) chosen[i] = (short)chosen_expert(c, i / top, i % top, top);
  __syncthreads();
  for (int e0 = 0; e0 < E; e0 += WARPS * 32) {               // a thread looks for its expert among the choices
    const int e = e0 + tid;
    if (e >= E) continue;
    bool any = false;
#pragma unroll
    for (int i = 0; i < NT * 8; ++i) slot_of[e][i] = -1;
    for (int i = 0; i < M * top; ++i)
      if (chosen[i] == e) { slot_of[e][i / top] = (signed char)(i % top); any = true; }
    picked[e] = any;
  }
  __syncthreads();
  if (warp == 0) {                                           // the experts that some token chose, in order
    int have = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const bool any = e0 + lane < E && picked[e0 + lane];
      const unsigned who = __ballot_sync(0xffffffffu, any);
      if (any) active[have + __popc(who & ((1u << lane) - 1u))] = (short)(e0 + lane);
      have += __popc(who);
    }
    if (lane == 0) n_active = have;
  }
  __syncthreads();
  // the walk: groups of 32 units (an expert's last one may be short), active experts one after another, then the shared one
  const int ge = (ff + 31) / 32, gs = (fs + 31) / 32;
  const int total = n_active * ge + gs;
  const int runs = slices * WARPS, run = slice * WARPS + warp;
  const int begin = (int)((long long)total * run / runs), end = (int)((long long)total * (run + 1) / runs);
  const size_t lo = min(n0 + g, N - 1), hi = min(n0 + g + 8, N - 1);      // rows past N read row N - 1 again, unstored
  const int row_len = top * ff + fs;
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  bool waited = false;
  for (int at = begin; at < end;) {
    // the part of this run that lies in one expert: groups g0 .. g1 of its `len` units
    const int ai = min(at / ge, n_active);
    const bool sh = ai == n_active;
    const int len = sh ? fs : ff;
    const int g0 = at - ai * ge, g1 = min(end - ai * ge, sh ? gs : ge);
    const bf16* w = sh ? Ws : W + (size_t)active[ai] * N * ff;
    const bf16 *w_lo = w + lo * len, *w_hi = w + hi * len;
    const bf16* x_row[NT];
    bool x_ok[NT];
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int tok = i * 8 + g;
      const int slot = sh ? (tok < M ? top : -1) : slot_of[active[ai]][tok];
      x_ok[i] = slot >= 0;
      x_row[i] = act + (x_ok[i] ? (size_t)tok * row_len + (size_t)slot * ff : 0);
    }
    for (int grp = g0; grp < g1; grp += MG_U) {
      uint4 wl[MG_U], wh[MG_U];
#pragma unroll
      for (int u = 0; u < MG_U; ++u) {
        const int k = (grp + u) * 32 + t * 8;
        wl[u] = wh[u] = make_uint4(0, 0, 0, 0);
        if (grp + u < g1 && k < len) {
          wl[u] = mg_stream(w_lo + k);
          wh[u] = mg_stream(w_hi + k);
        }
      }
      if (!waited) { pdl_wait(); pdl_trigger(); waited = true; }
#pragma unroll
      for (int u0 = 0; u0 < MG_U; u0 += 4) {
        uint4 xv[4][NT];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int k = (grp + u0 + u) * 32 + t * 8;
          const bool in = grp + u0 + u < g1 && k < len;
#pragma unroll
          for (int i = 0; i < NT; ++i) xv[u][i] = (in && x_ok[i]) ? mg_act(x_row[i] + k) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
          for (int i = 0; i < NT; ++i) {
            mg_mma(acc[i], wl[u0 + u].x, wh[u0 + u].x, wl[u0 + u].y, wh[u0 + u].y, xv[u][i].x, xv[u][i].y);
            mg_mma(acc[i], wl[u0 + u].z, wh[u0 + u].z, wl[u0 + u].w, wh[u0 + u].w, xv[u][i].z, xv[u][i].w);
          }
      }
    }
    at = ai * ge + g1;
  }
  if (!waited) { pdl_wait(); pdl_trigger(); }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) red[warp][i][lane][j] = acc[i][j];
  __syncthreads();
  const bool finisher = tid < NT * 32;
  const int i = tid >> 5;
  float s[4] = {0.f, 0.f, 0.f, 0.f};
  if (finisher) {
#pragma unroll
    for (int w = 0; w < WARPS; ++w)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[j] += red[w][i][lane][j];
  }
  if (slices > 1) {
    cg::cluster_group cluster = cg::this_cluster();
    if (finisher && slice > 0)
#pragma unroll
      for (int j = 0; j < 4; ++j) tile[i][lane][j] = s[j];
    cluster.sync();
    if (finisher && slice == 0)
      for (int q = 1; q < slices; ++q) {
        const float* other = cluster.map_shared_rank(&tile[0][0][0], q) + (i * 32 + lane) * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j) s[j] += other[j];
      }
    cluster.sync();                  // nobody leaves while the first CTA still reads its shared memory
    if (slice > 0) return;
  }
  if (!finisher) return;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int row = n0 + g + (j < 2 ? 0 : 8), tok = i * 8 + 2 * t + (j & 1);
    if (row < N && tok < M) out[(size_t)tok * N + row] = s[j];
  }
}

AB_API int ab_moe_gemv_max_tokens() { return MG_MAX_TOKENS; }
AB_API int ab_moe_gemv_max_experts() { return MG_MAX_EXPERTS; }

// Without `gated`, gate_up holds the up-projections alone, [E * ff, width] (ff and fs multiples of 16).
// act: scratch bfloat16 [M, top * ff + fs]; out: float32 [M, width].  `slices` (1, 2, 4 or 8): CTAs per 16 output columns.
AB_API int ab_moe_gemv_max_top() { return MG_MAX_TOP; }
AB_API int ab_moe_gemv(const void* h, const void* gate_up, const void* down, const void* gate_up_s, const void* down_s, const int* idx, const float* wts, const int* table,
                       const int* tokens, float weight, const float* z, void* act, float* out, int M, int top, int width, int ff,
                       int fs, int E, int activation, int gated, int weight_in, int slices, cudaStream_t stream) {
  if (M <= 0) return AB_OK;
  const Choice c{idx, wts, table, tokens, weight};
  if (M > MG_MAX_TOKENS || E <= 0 || E > MG_MAX_EXPERTS || top <= 0 || top > MG_MAX_TOP || top > E || width <= 0 || width % 8 || ff <= 0 ||
      ff % 8 || fs < 0 || fs % 8 || activation < 0 || activation >= MOE_ACT_KINDS || !choice_ok(c) || (fs > 0 && (!gate_up_s || !down_s)) ||
      (!gated && (ff % 16 || fs % 16)))
    return AB_BAD_ARG;
  if (slices != 1 && slices != 2 && slices != 4 && slices != 8) return AB_BAD_ARG;
  if ((((uintptr_t)h) | ((uintptr_t)gate_up) | ((uintptr_t)down) | ((uintptr_t)gate_up_s) | ((uintptr_t)down_s) |
       ((uintptr_t)act)) & 15) return AB_BAD_ARG;
  const int units = gated ? 8 : 16;
  const unsigned up_blocks = (unsigned)(E * (ff / units) + fs / units);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)((width + 15) / 16), (unsigned)slices);
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  int n_attr = 0;
  if (ab_pdl_enabled() && !ab_pdl_held) {
    attr[n_attr].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n_attr].val.programmaticStreamSerializationAllowed = 1;
    ++n_attr;
  }
  if (slices > 1) {
    attr[n_attr].id = cudaLaunchAttributeClusterDimension;
    attr[n_attr].val.clusterDim.x = 1;
    attr[n_attr].val.clusterDim.y = (unsigned)slices;
    attr[n_attr].val.clusterDim.z = 1;
    ++n_attr;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n_attr;
  cudaError_t e = cudaSuccess;
#define AB_GO(NT, WARPS)                                                                                               \
  {                                                                                                                    \
    ab_launch(gated ? moe_gemv_up_kernel<NT, true> : moe_gemv_up_kernel<NT, false>, dim3(up_blocks), dim3(256), 0, stream, \
              (const bf16*)h, (const bf16*)gate_up, (const bf16*)gate_up_s, c, z, (bf16*)act, M, width, top, ff, fs, E,   \
              activation, weight_in);                                                                                  \
    cfg.blockDim = dim3(WARPS * 32);                                                                                   \
    e = cudaLaunchKernelEx(&cfg, moe_gemv_down_kernel<NT, WARPS>, (const bf16*)act, (const bf16*)down, (const bf16*)down_s, c, out, \
                           M, width, top, ff, fs, E, slices);                                                                         \
  }
  if (M <= 8) AB_GO(1, 16)
  else if (M <= 16) AB_GO(2, 16)
  else AB_GO(4, 8)
#undef AB_GO
  if (e != cudaSuccess) return AB_CUDA_ERR + (int)e;
  return ab_launch_status();
}

// A state-space mixer with one decay and one step size per head and token (Dao and Gu, "Transformers are SSMs:
// Generalized Models and Efficient Algorithms Through Structured State Space Duality").
//
// A token's projected row (float32) holds [z | x | B | C | dt]: z and x H heads of V, B and C G groups of N, dt H numbers.
//   x, B, C  pass a causal convolution per channel over `taps` tokens (with a bias) and SiLU; a sequence's last taps - 1
//            inputs are state
//   dt       softplus(dt + bias_h);   a = exp(-exp(A_log_h) dt)                 head h reads group h // (H / G)
//   S        <- a S + dt B x^T   [N, V] float32 per (sequence, head);   y = S^T C + skip_h x
//   out      = (y silu(z)) in `parts` equal parts, each divided by its own root mean square, times w
//
// Three forms of the recurrence, the same sums up to rounding:
//   ssm_step    one token per sequence: convolution, step size, decay, update and read-out in one kernel.  A CTA takes a
//               (sequence, head, tile of value columns); the tile of S is asked for, 16 bytes per thread and row, before the
//               wait for the projection, and goes back once.
//   ssm_chunks  prompts in bfloat16: 64 tokens at a time on the tensor cores (mma.sync), S in the accumulators of a CTA that
//               walks one sequence's chunks for one (head, tile of columns).  With L_t the running sum of the chunk's log
//               decays,  y_t = exp(L_t) S^T C_t + sum_(s <= t) exp(L_t - L_s) dt_s (C_t . B_s) x_s  and
//               S <- exp(L_end) S + sum_s exp(L_end - L_s) dt_s B_s x_s^T.  B, C and x are the convolution's outputs rounded
//               to bfloat16; everything else that meets them (S, the weights of the scores, the weighted x) is split into
//               two bfloat16 numbers, high and low, and multiplied twice, so that it enters with 16 bits.
//   otherwise   ssm_prepare leaves float32 rows and the walk of csrc/gated_recurrence.cu (mode 2) does the rest.
// Around them: ssm_prepare (convolution, step sizes, decays for many tokens), ssm_gate_norm (the gate and the norm; after
// ssm_step it moves the convolution's inputs on, since every CTA of that kernel has read them by then).
#include "attention_common.cuh"
#include "launch.cuh"

#define SSM_MAX_TAPS 17
#define SSM_RUN 8            // tokens that a thread of ssm_prepare walks

__device__ __forceinline__ float ssm_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float ssm_silu(float x) { return x / (1.0f + expf(-x)); }

struct SsmSizes {
  int H, G, N, V, taps;
  __host__ __device__ int inner() const { return H * V; }
  __host__ __device__ int channels() const { return H * V + 2 * G * N; }      // x | B | C, convolved
  __host__ __device__ int off_x() const { return H * V; }
  __host__ __device__ int off_dt() const { return 2 * H * V + 2 * G * N; }
};

template <int W> struct Lanes { float v[W]; };
template <int W> __device__ __forceinline__ Lanes<W> load_lanes(const float* p) {
  Lanes<W> r;
  if (W == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    r.v[0] = q.x; r.v[1 % W] = q.y; r.v[2 % W] = q.z; r.v[3 % W] = q.w;
  } else r.v[0] = *p;
  return r;
}
template <int W> __device__ __forceinline__ void store_lanes(float* p, const Lanes<W>& r) {
  if (W == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1 % W], r.v[2 % W], r.v[3 % W]);
  else *p = r.v[0];
}
template <int W> __device__ __forceinline__ void store_lanes(bf16* p, const Lanes<W>& r) {
  if (W == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(r.v[0], r.v[1 % W]), pack_bf16(r.v[2 % W], r.v[3 % W]));
  else *p = __float2bfloat16_rn(r.v[0]);
}

// ---------------------------------------------------------------------------
// many tokens: convolution, step sizes, decays
// ---------------------------------------------------------------------------
// A thread takes W neighbouring channels of SSM_RUN tokens (blocks with blockIdx.y < chan_blocks) or the heads' numbers.
// K > 0: the number of taps, the last K - 1 inputs in registers; K = 0: any number, inputs fetched per tap.
// conv_w is [taps, channels]; conv_state [slots, taps - 1, channels], oldest first.
template <typename TO, int W, int K>
__global__ void __launch_bounds__(128)
ssm_prepare_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
                   const float* __restrict__ conv_state, const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                   TO* __restrict__ xbc, float* __restrict__ decay, float* __restrict__ dt, int log_decay,
                   const int* __restrict__ tok_seq, const int* __restrict__ cu_q, const int* __restrict__ slots,
                   int n_tokens, SsmSizes z, int chan_blocks) {
  pdl_wait();
  pdl_trigger();
  const int t0 = blockIdx.x * SSM_RUN, t1 = min(n_tokens, t0 + SSM_RUN);
  const int Cc = z.channels(), taps = K ? K : z.taps;
  if ((int)blockIdx.y >= chan_blocks) {
    const int h = (blockIdx.y - chan_blocks) * blockDim.x + threadIdx.x;
    if (h >= z.H) return;
    const float ea = expf(A_log[h]), bias = dt_bias[h];
    for (int t = t0; t < t1; ++t) {
      if (tok_seq[t] < 0) continue;
      const float d = ssm_softplus(proj[(size_t)t * ld + z.off_dt() + h] + bias);
      dt[(size_t)t * z.H + h] = d;
      decay[(size_t)t * z.H + h] = log_decay ? -ea * d : expf(-ea * d);
    }
    return;
  }
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * W;
  if (c >= Cc) return;
  const float* x = proj + z.off_x() + c;
  const Lanes<W> bias = load_lanes<W>(conv_b + c);
  Lanes<W> w[K ? K : 1], past[K > 1 ? K - 1 : 1];
#pragma unroll
  for (int j = 0; j < K; ++j) w[j] = load_lanes<W>(conv_w + (size_t)j * Cc + c);
  for (int t = t0; t < t1; ++t) {
    const int b = tok_seq[t];
    if (b < 0) continue;
    const int i = t - cu_q[b];
    const float* held = conv_state + (size_t)slots[b] * (taps - 1) * Cc + c;
    if (K) {
      if (t == t0 || i == 0) {
#pragma unroll
        for (int j = 0; j < K - 1; ++j) {
          const int src = i - (K - 1) + j;
          past[j] = src >= 0 ? load_lanes<W>(x + (size_t)(t - (K - 1) + j) * ld) : load_lanes<W>(held + (size_t)(K - 1 + src) * Cc);
        }
      }
    }
    const Lanes<W> now = load_lanes<W>(x + (size_t)t * ld);
    Lanes<W> acc = bias;
    if (K) {
#pragma unroll
      for (int j = 0; j < K - 1; ++j)
#pragma unroll
        for (int e = 0; e < W; ++e) acc.v[e] = fmaf(w[j].v[e], past[j].v[e], acc.v[e]);
#pragma unroll
      for (int e = 0; e < W; ++e) acc.v[e] = fmaf(w[K ? K - 1 : 0].v[e], now.v[e], acc.v[e]);
#pragma unroll
      for (int j = 0; j + 1 < K - 1; ++j) past[j] = past[j + 1];
      if (K > 1) past[K > 1 ? K - 2 : 0] = now;
    } else {
      for (int j = 0; j < taps; ++j) {
        const int src = i - (taps - 1) + j;
        const Lanes<W> in = src >= 0 ? load_lanes<W>(x + (size_t)(t - (taps - 1) + j) * ld)
                                     : load_lanes<W>(held + (size_t)(taps - 1 + src) * Cc);
        const Lanes<W> wj = load_lanes<W>(conv_w + (size_t)j * Cc + c);
#pragma unroll
        for (int e = 0; e < W; ++e) acc.v[e] = fmaf(wj.v[e], in.v[e], acc.v[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < W; ++e) acc.v[e] = ssm_silu(acc.v[e]);
    store_lanes<W>(xbc + (size_t)t * Cc + c, acc);
  }
}

// conv_state[slot] <- the sequence's last taps - 1 inputs: a thread per (sequence, channel) reads what it keeps first
__global__ void ssm_conv_move_kernel(const float* __restrict__ proj, int ld, float* __restrict__ conv_state,
                                     const int* __restrict__ cu_q, const int* __restrict__ slots, int n_seqs, SsmSizes z) {
  pdl_wait();
  pdl_trigger();
  const int Cc = z.channels(), keep = z.taps - 1;
  const long long id = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (id >= (long long)n_seqs * Cc) return;
  const int b = (int)(id / Cc), c = (int)(id - (long long)b * Cc);
  const int slot = slots[b];
  if (slot < 0) return;
  const int t0 = cu_q[b], n = cu_q[b + 1] - t0;
  const float* x = proj + z.off_x() + c;
  float* held = conv_state + (size_t)slot * keep * Cc + c;
  float now[SSM_MAX_TAPS - 1];
#pragma unroll
  for (int s = 0; s < SSM_MAX_TAPS - 1; ++s)
    if (s < keep) {
      const int i = n - keep + s;
      now[s] = i >= 0 ? x[(size_t)(t0 + i) * ld] : held[(size_t)(s + n) * Cc];
    }
#pragma unroll
  for (int s = 0; s < SSM_MAX_TAPS - 1; ++s)
    if (s < keep) held[(size_t)s * Cc] = now[s];
}

static bool ssm_sizes_ok(const SsmSizes& z) {
  return z.H > 0 && z.G > 0 && z.H % z.G == 0 && z.N > 0 && z.N <= 256 && z.V > 0 && z.taps >= 1 && z.taps <= SSM_MAX_TAPS;
}

// xbc [T, channels] float32 or bfloat16; decay, dt [T, H] float32 (decay: exp(..), or its logarithm with `log_decay`)
AB_API int ab_ssm_prepare(const float* proj, int ld, const float* conv_w, const float* conv_b, float* conv_state,
                          const float* A_log, const float* dt_bias, void* xbc, int xbc_dtype, float* decay, float* dt,
                          int log_decay, const int* tok_seq, const int* cu_q, const int* slots, int n_tokens, int n_seqs,
                          int H, int G, int N, int V, int taps, int write_state, cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  const SsmSizes z{H, G, N, V, taps};
  if (!ssm_sizes_ok(z) || !proj || !conv_w || !conv_b || !A_log || !dt_bias || !xbc || !decay || !dt || (taps > 1 && !conv_state))
    return AB_BAD_ARG;
  const int Cc = z.channels();
  auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = Cc % 4 == 0 && ld % 4 == 0 && z.off_x() % 4 == 0 && al(proj) && al(conv_w) && al(conv_b) && al(conv_state) && al(xbc);
  const int per = 128 * (vec ? 4 : 1), chan_blocks = (Cc + per - 1) / per;
  const dim3 grid((unsigned)((n_tokens + SSM_RUN - 1) / SSM_RUN), (unsigned)(chan_blocks + (H + 127) / 128));
#define AB_GO(TO, W, K)                                                                                                \
  ab_launch(ssm_prepare_kernel<TO, W, K>, grid, dim3(128), 0, stream, proj, ld, conv_w, conv_b, (const float*)conv_state, \
            A_log, dt_bias, (TO*)xbc, decay, dt, log_decay, tok_seq, cu_q, slots, n_tokens, z, chan_blocks)
#define AB_K(TO, W)                                                                                                    \
  {                                                                                                                    \
    if (taps == 2) AB_GO(TO, W, 2); else if (taps == 3) AB_GO(TO, W, 3); else if (taps == 4) AB_GO(TO, W, 4);          \
    else AB_GO(TO, W, 0);                                                                                              \
  }
  if (xbc_dtype == AB_F32) { if (vec) AB_K(float, 4) else AB_K(float, 1) }
  else if (xbc_dtype == AB_BF16) { if (vec) AB_K(bf16, 4) else AB_K(bf16, 1) }
  else return AB_BAD_ARG;
#undef AB_K
#undef AB_GO
  int rc = ab_launch_status();
  if (rc || !write_state || taps == 1) return rc;
  const long long total = (long long)n_seqs * Cc;
  ab_launch(ssm_conv_move_kernel, dim3((unsigned)((total + 127) / 128)), dim3(128), 0, stream, proj, ld, conv_state, cu_q,
            slots, n_seqs, z);
  return ab_launch_status();
}

// ---------------------------------------------------------------------------
// one token per sequence
// ---------------------------------------------------------------------------
// 256 threads: CV / 4 of them side by side on a row of the tile, R rows each.  What a thread asks for before the wait (the
// tile of S, the convolution's kept inputs and weights) was written a step ago or never.
template <int CV, int R>
__global__ void __launch_bounds__(256)
ssm_step_kernel(const float* __restrict__ proj, int ld, const float* __restrict__ conv_w, const float* __restrict__ conv_b,
                const float* __restrict__ conv_state, const float* __restrict__ A_log, const float* __restrict__ dt_bias,
                const float* __restrict__ skip, float* __restrict__ state, float* __restrict__ y,
                const int* __restrict__ tok_seq, const int* __restrict__ slots, SsmSizes z, int write_state) {
  constexpr int C4 = CV / 4, RS = 256 / C4, MAXC = (512 + CV + 255) / 256;
  __shared__ __align__(16) float row[512 + CV];          // B | C | x of this CTA, after convolution and SiLU
  __shared__ __align__(16) float red[8][CV];
  const int t = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * CV;
  const int N = z.N, V = z.V, Cc = z.channels(), taps = z.taps;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int b = tok_seq[t];
  float* yr = y + (size_t)t * z.inner() + (size_t)h * V + col0;
  const int cw = min(CV, V - col0);
  if (b < 0) {
    pdl_wait();
    pdl_trigger();
    for (int j = tid; j < cw; j += 256) yr[j] = 0.f;
    return;
  }
  const int slot = slots[b];
  const int c4 = (tid % C4) * 4, r0 = tid / C4;
  const bool col_ok = c4 < cw;
  float* st = state + (((size_t)slot * z.H + h) * N) * V + col0 + c4;
  float4 S[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int n = r0 + i * RS;
    S[i] = (n < N && col_ok) ? *reinterpret_cast<const float4*>(st + (size_t)n * V) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const int g = h / (z.H / z.G), n_ch = 2 * N + cw;
  const float* held = conv_state + (size_t)slot * (taps - 1) * Cc;
  int ch[MAXC];
  float acc[MAXC], last[MAXC];
#pragma unroll
  for (int k = 0; k < MAXC; ++k) {
    const int i = tid + k * 256;
    ch[k] = -1;
    if (i < n_ch) {
      const int c = i < N ? z.inner() + g * N + i : i < 2 * N ? z.inner() + z.G * N + g * N + i - N : h * V + col0 + i - 2 * N;
      ch[k] = c;
      acc[k] = conv_b[c];
      for (int j = 0; j < taps - 1; ++j) acc[k] = fmaf(conv_w[(size_t)j * Cc + c], held[(size_t)j * Cc + c], acc[k]);
      last[k] = conv_w[(size_t)(taps - 1) * Cc + c];
    }
  }
  const float ea = expf(A_log[h]), bias = dt_bias[h], sk = skip[h];
  pdl_wait();
  pdl_trigger();
  const float* p = proj + (size_t)t * ld;
  const float raw_dt = p[z.off_dt() + h];
#pragma unroll
  for (int k = 0; k < MAXC; ++k)
    if (ch[k] >= 0) row[tid + k * 256] = ssm_silu(fmaf(last[k], p[z.off_x() + ch[k]], acc[k]));
  const float dt = ssm_softplus(raw_dt + bias), a = expf(-ea * dt);
  __syncthreads();
  const float* xs = row + 2 * N;
  float4 x4 = make_float4(0.f, 0.f, 0.f, 0.f);
  if (col_ok) x4 = make_float4(xs[c4] * dt, xs[c4 + 1] * dt, xs[c4 + 2] * dt, xs[c4 + 3] * dt);
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int n = r0 + i * RS;
    if (n < N) {
      const float kb = row[n], qc = row[N + n];
      S[i].x = fmaf(a, S[i].x, kb * x4.x);
      S[i].y = fmaf(a, S[i].y, kb * x4.y);
      S[i].z = fmaf(a, S[i].z, kb * x4.z);
      S[i].w = fmaf(a, S[i].w, kb * x4.w);
      o.x = fmaf(S[i].x, qc, o.x);
      o.y = fmaf(S[i].y, qc, o.y);
      o.z = fmaf(S[i].z, qc, o.z);
      o.w = fmaf(S[i].w, qc, o.w);
      if (write_state && col_ok) *reinterpret_cast<float4*>(st + (size_t)n * V) = S[i];
    }
  }
#pragma unroll
  for (int d = C4; d < 32; d <<= 1) {
    o.x += __shfl_xor_sync(0xffffffffu, o.x, d);
    o.y += __shfl_xor_sync(0xffffffffu, o.y, d);
    o.z += __shfl_xor_sync(0xffffffffu, o.z, d);
    o.w += __shfl_xor_sync(0xffffffffu, o.w, d);
  }
  if (lane < C4) *reinterpret_cast<float4*>(&red[warp][c4]) = o;
  __syncthreads();
  if (tid < cw) {
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) s += red[w][tid];
    yr[tid] = fmaf(sk, xs[tid], s);
  }
}

// 1 if ssm_step takes the sizes: value sizes in steps of 4
AB_API int ab_ssm_step_supports(int N, int V) { return N > 0 && N <= 256 && V > 0 && V % 4 == 0 ? 1 : 0; }

// `cols`: value columns per CTA (16, 32 or 64).  The convolution's kept inputs are left as they are (ab_ssm_gate_norm
// moves them on).
AB_API int ab_ssm_step(const float* proj, int ld, const float* conv_w, const float* conv_b, const float* conv_state,
                       const float* A_log, const float* dt_bias, const float* skip, float* state, float* y,
                       const int* tok_seq, const int* slots, int n_tokens, int H, int G, int N, int V, int taps, int cols,
                       int write_state, cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  const SsmSizes z{H, G, N, V, taps};
  if (!ssm_sizes_ok(z) || !ab_ssm_step_supports(N, V) || H > 65535 || (((uintptr_t)state) & 15)) return AB_BAD_ARG;
  const dim3 grid((unsigned)n_tokens, (unsigned)H, (unsigned)((V + cols - 1) / cols));
#define AB_GO(CV, R)                                                                                                   \
  ab_launch(ssm_step_kernel<CV, R>, grid, dim3(256), 0, stream, proj, ld, conv_w, conv_b, conv_state, A_log, dt_bias, skip, \
            state, y, tok_seq, slots, z, write_state)
  if (cols == 64) {
    if (N <= 16) AB_GO(64, 1); else if (N <= 32) AB_GO(64, 2); else if (N <= 64) AB_GO(64, 4);
    else if (N <= 128) AB_GO(64, 8); else AB_GO(64, 16);
  } else if (cols == 32) {
    if (N <= 32) AB_GO(32, 1); else if (N <= 64) AB_GO(32, 2); else if (N <= 128) AB_GO(32, 4); else AB_GO(32, 8);
  } else if (cols == 16) {
    if (N <= 64) AB_GO(16, 1); else if (N <= 128) AB_GO(16, 2); else AB_GO(16, 4);
  } else
    return AB_BAD_ARG;
#undef AB_GO
  return ab_launch_status();
}

// ---------------------------------------------------------------------------
// gate and norm
// ---------------------------------------------------------------------------
// A block per (token, part): out = cast(u / rms(u) * w), u = y silu(z), over the part's n numbers.  NV > 0: n and the row
// strides are multiples of 4 and the part fits NV quads per thread; NV = 0: any size, u formed twice.
// `conv_state` (or null): the token's convolution inputs become the newest of what its sequence keeps (one token per
// sequence), by the blocks behind a token's parts.  What is asked for before the wait is older than the kernel before.
template <typename TO, int NV>
__global__ void __launch_bounds__(512)
ssm_gate_norm_kernel(const float* __restrict__ y, const float* __restrict__ proj, int ld, const float* __restrict__ w,
                     TO* __restrict__ out, float* __restrict__ conv_state, const int* __restrict__ tok_seq,
                     const int* __restrict__ slots, int n, float eps, int parts, SsmSizes z) {
  __shared__ float scratch[32];
  const int t = blockIdx.x, base = blockIdx.y * n;
  const int b = tok_seq[t];
  if ((int)blockIdx.y >= parts) {
    const int Cc = z.channels(), keep = z.taps - 1, c = ((int)blockIdx.y - parts) * blockDim.x + threadIdx.x;
    float* held = conv_state + (b < 0 ? 0 : (size_t)slots[b] * keep * Cc) + c;
    float now[SSM_MAX_TAPS - 1];
    if (b >= 0 && c < Cc) {
#pragma unroll
      for (int s = 0; s < SSM_MAX_TAPS - 1; ++s)
        if (s < keep) now[s] = s + 1 < keep ? held[(size_t)(s + 1) * Cc] : proj[(size_t)t * ld + z.off_x() + c];
    }
    pdl_wait();
    pdl_trigger();
    if (b >= 0 && c < Cc) {
#pragma unroll
      for (int s = 0; s < SSM_MAX_TAPS - 1; ++s)
        if (s < keep) held[(size_t)s * Cc] = now[s];
    }
    return;
  }
  TO* o = out + (size_t)t * z.inner() + base;
  if (b < 0) {
    pdl_wait();
    pdl_trigger();
    for (int j = threadIdx.x; j < n; j += blockDim.x) o[j] = from_f32<TO>(0.f);
    return;
  }
  const float* yr = y + (size_t)t * z.inner() + base;
  const float* zr = proj + (size_t)t * ld + base;
  const float* wr = w + base;
  float ss = 0.f;
  if (NV > 0) {
    Lanes<4> u[NV > 0 ? NV : 1], wv[NV > 0 ? NV : 1], gv[NV > 0 ? NV : 1];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int j = (threadIdx.x + k * blockDim.x) * 4;
      if (j < n) {
        gv[k] = load_lanes<4>(zr + j);
        wv[k] = load_lanes<4>(wr + j);
      }
    }
    pdl_wait();
    pdl_trigger();
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int j = (threadIdx.x + k * blockDim.x) * 4;
      if (j < n) u[k] = load_lanes<4>(yr + j);
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      if ((threadIdx.x + k * blockDim.x) * 4 < n) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          u[k].v[e] *= ssm_silu(gv[k].v[e]);
          ss += u[k].v[e] * u[k].v[e];
        }
      }
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)n + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int j = (threadIdx.x + k * blockDim.x) * 4;
      if (j < n) {
#pragma unroll
        for (int e = 0; e < 4; ++e) u[k].v[e] *= inv * wv[k].v[e];
        store_lanes<4>(o + j, u[k]);
      }
    }
  } else {
    pdl_wait();
    pdl_trigger();
    for (int j = threadIdx.x; j < n; j += blockDim.x) {
      const float u = yr[j] * ssm_silu(zr[j]);
      ss += u * u;
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)n + eps);
    for (int j = threadIdx.x; j < n; j += blockDim.x) o[j] = from_f32<TO>(yr[j] * ssm_silu(zr[j]) * (inv * wr[j]));
  }
}

AB_API int ab_ssm_gate_norm(const float* y, const float* proj, int ld, const float* w, void* out, int out_dtype,
                            float* conv_state, const int* tok_seq, const int* slots, int n_tokens, int parts, float eps,
                            int H, int G, int N, int V, int taps, cudaStream_t stream) {
  if (n_tokens <= 0) return AB_OK;
  const SsmSizes z{H, G, N, V, taps};
  if (!ssm_sizes_ok(z) || parts <= 0 || z.inner() % parts || parts > 32767 || (taps == 1 && conv_state)) return AB_BAD_ARG;
  const int n = z.inner() / parts;
  auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = n % 4 == 0 && ld % 4 == 0 && al(y) && al(proj) && al(w) && al(out) && n <= 512 * 4 * 4;
  const int threads = n >= 4096 ? 512 : n >= 1024 ? 256 : n >= 256 ? 128 : 64;
  const int nv = vec ? (n / 4 + threads - 1) / threads : 0;
  const int movers = conv_state != nullptr ? (z.channels() + threads - 1) / threads : 0;
  const dim3 grid((unsigned)n_tokens, (unsigned)(parts + movers));
#define AB_GO(TO, NV)                                                                                                  \
  ab_launch(ssm_gate_norm_kernel<TO, NV>, grid, dim3(threads), 0, stream, y, proj, ld, w, (TO*)out, conv_state, tok_seq, slots, \
            n, eps, parts, z)
#define AB_NV(TO)                                                                                                      \
  { if (nv == 0) AB_GO(TO, 0); else if (nv == 1) AB_GO(TO, 1); else if (nv == 2) AB_GO(TO, 2); else AB_GO(TO, 4); }
  if (out_dtype == AB_F32) AB_NV(float)
  else if (out_dtype == AB_BF16) AB_NV(bf16)
  else return AB_BAD_ARG;
#undef AB_NV
#undef AB_GO
  return ab_launch_status();
}

// ---------------------------------------------------------------------------
// prompts: chunks of 64 tokens on the tensor cores
// ---------------------------------------------------------------------------
#define SC_T 64

__device__ __forceinline__ void sc_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(smem_u32(dst)), "l"(src));
}
// v = hi + lo up to 2^-17: two bfloat16 numbers each
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}

#define SC_CV 32               // value columns per CTA
#define SC_PV (SC_CV + 8)      // pitch of rows of value columns
#define SC_PP (SC_T + 8)       // pitch of rows of weights
#define SC_WORKERS 512         // threads that hold S and outputs; one more warp forms the scales
#define SC_THREADS (SC_WORKERS + 32)

// What a chunk's step sizes and log decays come to, in powers of two: L_t, the running sum of the log decays (times log2 e).
struct ChunkScales {
  float L[SC_T];          // L_t
  float q[SC_T];          // L_s - log2 dt_s: a key's score is multiplied by 2^(L_t - q_s)
  float e[SC_T];          // 2^(L_t)
  float w[SC_T];          // 2^(L_end - L_s) dt_s
  float end[4];           // 2^(L_end)
};

static size_t chunk_smem(int N) {
  return sizeof(bf16) * (4 * (size_t)SC_T * (N + 8) + 2 * (size_t)SC_T * SC_PV + 2 * (size_t)N * SC_PV + 2 * (size_t)SC_T * SC_PV +
                         2 * (size_t)SC_T * SC_PP) + 2 * sizeof(ChunkScales);
}

// Sixteen warps.  Warp w takes tokens 16 (w / 4) .. + 15 of the chunk and, of them, the scores against tokens 16 (w % 4) .. + 15
// and the output columns 8 (w % 4) .. + 7; of S the row tiles w % 8, w % 8 + 8, .. (RT of them) and columns 16 (w / 8) .. + 15.
// A seventeenth warp forms the next chunk's scales.  Two barriers per chunk: (1) S and the weighted x of the chunk lie in
// shared memory, split; (2) so do the weights of its scores, and the next chunk's rows and scales have arrived.
template <int RT>
__global__ void __launch_bounds__(SC_THREADS)
ssm_chunks_kernel(const bf16* __restrict__ xbc, const float* __restrict__ la, const float* __restrict__ dt,
                  const float* __restrict__ skip, float* __restrict__ state, float* __restrict__ y,
                  const int* __restrict__ cu_q, const int* __restrict__ slots, SsmSizes z, int write_state) {
  extern __shared__ __align__(16) unsigned char sm[];
  const int N = z.N, V = z.V, H = z.H, Cc = z.channels(), PN = N + 8;
  bf16* Bs = reinterpret_cast<bf16*>(sm);                       // [2][64][PN]
  bf16* Cs = Bs + 2 * SC_T * PN;                                // [2][64][PN]
  bf16* xs = Cs + 2 * SC_T * PN;                                // [2][64][PV]
  bf16* Sh = xs + 2 * SC_T * SC_PV;                             // [N][PV] the state before the chunk, high and low parts
  bf16* Sl = Sh + N * SC_PV;
  bf16* wh = Sl + N * SC_PV;                                    // [64][PV] w_s x_s
  bf16* wl = wh + SC_T * SC_PV;
  bf16* Ph = wl + SC_T * SC_PV;                                 // [64][PP] scores times their weights
  bf16* Pl = Ph + SC_T * SC_PP;
  ChunkScales* scales = reinterpret_cast<ChunkScales*>(Pl + SC_T * SC_PP);      // [2]
  const int b = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * SC_CV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t4 = lane & 3;
  const int slot = slots[b], t0 = cu_q[b], t1 = cu_q[b + 1];
  if (slot < 0 || t1 <= t0) { pdl_wait(); pdl_trigger(); return; }
  const int grp = h / (H / z.G);
  const int srow = (warp & 7) * 16, scol = ((warp >> 3) & 1) * 16;                    // this warp's part of S
  float* st = state + ((size_t)slot * H + h) * N * V + col0 + scol;
  float S[RT][2][4];
#pragma unroll
  for (int r = 0; r < RT; ++r)
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int n = srow + 128 * r + g, c = nt * 8 + 2 * t4;
      const bool in = warp < 16 && srow + 128 * r < N && col0 + scol + c < V;
      const float2 lo = in ? *reinterpret_cast<const float2*>(st + (size_t)n * V + c) : make_float2(0.f, 0.f);
      const float2 hi = in ? *reinterpret_cast<const float2*>(st + (size_t)(n + 8) * V + c) : make_float2(0.f, 0.f);
      S[r][nt][0] = lo.x; S[r][nt][1] = lo.y; S[r][nt][2] = hi.x; S[r][nt][3] = hi.y;
    }
  // who copies what of a chunk: a thread keeps its 16-byte column of B and C and walks down the rows; the first 256 one piece of x
  const int pn = N >> 3, per_pass = SC_WORKERS / pn, br = tid / pn, bc = (tid - br * pn) * 8;
  const bool worker = warp < 16, copies = worker && br < per_pass;
  const int xr = tid >> 2, xc = (tid & 3) * 8;
  pdl_wait();
  pdl_trigger();
  const float sk = skip[h];
  const bf16* Bg = xbc + z.inner() + (size_t)grp * N + bc;
  const bf16* xg = xbc + (size_t)h * V + col0 + xc;
  const size_t c_ahead = (size_t)z.G * N;
  auto load = [&](int buf, int c0) {
    const int n = min(SC_T, t1 - c0);
    if (copies) {
      const bf16* src = Bg + (size_t)(c0 + br) * Cc;
      bf16* db = Bs + (buf * SC_T + br) * PN + bc;
      for (int r = br; r < SC_T; r += per_pass, src += (size_t)per_pass * Cc, db += per_pass * PN) {
        bf16* dc = db + 2 * SC_T * PN;
        if (r < n) {
          sc_async16(db, src);
          sc_async16(dc, src + c_ahead);
        } else {
          *reinterpret_cast<uint4*>(db) = make_uint4(0, 0, 0, 0);
          *reinterpret_cast<uint4*>(dc) = make_uint4(0, 0, 0, 0);
        }
      }
    }
    if (tid < SC_T * (SC_CV / 8)) {
      bf16* d = xs + (buf * SC_T + xr) * SC_PV + xc;
      if (xr < n && col0 + xc < V) sc_async16(d, xg + (size_t)(c0 + xr) * Cc);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };
  // the last warp's lanes hold two tokens' numbers each; tokens past the end have no decay and no weight
  float l0 = 0.f, l1 = 0.f, d0 = 0.f, d1 = 0.f;
  auto fetch = [&](int c0) {
    const int a = c0 + 2 * lane;
    l0 = a < t1 ? la[(size_t)a * H + h] : 0.f;
    d0 = a < t1 ? dt[(size_t)a * H + h] : 0.f;
    l1 = a + 1 < t1 ? la[(size_t)(a + 1) * H + h] : 0.f;
    d1 = a + 1 < t1 ? dt[(size_t)(a + 1) * H + h] : 0.f;
  };
  auto scan = [&](ChunkScales& s) {
    const float v0 = l0 * LOG2E, v1 = l1 * LOG2E;
    float incl = v0 + v1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += up;
    }
    float before = __shfl_up_sync(0xffffffffu, incl, 1);
    if (lane == 0) before = 0.f;
    const float end = __shfl_sync(0xffffffffu, incl, 31), La = before + v0;
    *reinterpret_cast<float2*>(s.L + 2 * lane) = make_float2(La, incl);
    *reinterpret_cast<float2*>(s.q + 2 * lane) = make_float2(La - log2f(d0), incl - log2f(d1));
    *reinterpret_cast<float2*>(s.e + 2 * lane) = make_float2(fast_exp2(La), fast_exp2(incl));
    *reinterpret_cast<float2*>(s.w + 2 * lane) = make_float2(fast_exp2(end - La) * d0, fast_exp2(end - incl) * d1);
    if (lane == 0) s.end[0] = fast_exp2(end);
  };
  const int a_row = (lane & 7) + ((lane >> 3) & 1) * 8, a_col = (lane >> 4) * 8;       // first operand, rows of k
  const int b_row = (lane & 7) + (lane >> 4) * 8, b_col = ((lane >> 3) & 1) * 8;       // second operand, rows of k
  const int mi = (warp >> 2) & 3, mj = warp & 3, m0 = mi * 16;                         // tokens; scores' tokens and columns
  // shared-memory addresses of this lane's matrix rows, in bytes, without what moves with the loops
  const uint32_t aC = smem_u32(Cs + (m0 + a_row) * PN + a_col), aB = smem_u32(Bs + (mj * 16 + b_row) * PN + b_col);
  const uint32_t aS = smem_u32((lane < 16 ? Sh : Sl) + a_row * SC_PV + mj * 8);
  const uint32_t aBt = smem_u32(Bs + b_row * PN + srow + b_col);
  const uint32_t aW = smem_u32(wh + a_row * SC_PV + scol + a_col), to_wl = SC_T * SC_PV * 2;      // wl lies behind wh
  const uint32_t aP = smem_u32(Ph + (m0 + a_row) * SC_PP + a_col), to_pl = SC_T * SC_PP * 2;      // and Pl behind Ph
  const uint32_t aX = smem_u32(xs + lane * SC_PV + mj * 8);                            // 32 rows of x, eight columns
  const uint32_t bytes_bc = SC_T * PN * 2, bytes_x = SC_T * SC_PV * 2;                 // from one buffer to the other
  // S and the weighted x of the chunk in buffer `buf`, as pairs of bfloat16 numbers
  auto lay_out = [&](int buf) {
#pragma unroll
    for (int r = 0; r < RT; ++r) {
      if (srow + 128 * r < N) {
        const int at = (srow + 128 * r + g) * SC_PV + scol + 2 * t4;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          uint32_t hi, lo;
          split2(S[r][nt][0], S[r][nt][1], hi, lo);
          *reinterpret_cast<uint32_t*>(Sh + at + nt * 8) = hi;
          *reinterpret_cast<uint32_t*>(Sl + at + nt * 8) = lo;
          split2(S[r][nt][2], S[r][nt][3], hi, lo);
          *reinterpret_cast<uint32_t*>(Sh + at + 8 * SC_PV + nt * 8) = hi;
          *reinterpret_cast<uint32_t*>(Sl + at + 8 * SC_PV + nt * 8) = lo;
        }
      }
    }
    const int row = tid >> 3, c = (tid & 7) * 4;
    const uint2 v = *reinterpret_cast<const uint2*>(xs + (buf * SC_T + row) * SC_PV + c);
    const float w = scales[buf].w[row];
    uint2 hi, lo;
    split2(w * __uint_as_float(v.x << 16), w * __uint_as_float(v.x & 0xffff0000u), hi.x, lo.x);
    split2(w * __uint_as_float(v.y << 16), w * __uint_as_float(v.y & 0xffff0000u), hi.y, lo.y);
    *reinterpret_cast<uint2*>(wh + row * SC_PV + c) = hi;
    *reinterpret_cast<uint2*>(wl + row * SC_PV + c) = lo;
  };
  if (worker) {
    load(0, t0);
  } else {
    fetch(t0);
    scan(scales[0]);
    fetch(t0 + SC_T);
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  if (worker) lay_out(0);
  int buf = 0;
  for (int c0 = t0; c0 < t1; c0 += SC_T, buf ^= 1) {
    const bool more = c0 + SC_T < t1;
    float Y[4] = {0.f, 0.f, 0.f, 0.f}, Y2[4] = {0.f, 0.f, 0.f, 0.f};
    __syncthreads();                       // (1)
    if (!worker) {
      if (more) {
        scan(scales[buf ^ 1]);
        fetch(c0 + 2 * SC_T);
      }
    } else {
      if (more) load(buf ^ 1, c0 + SC_T);
      const ChunkScales& sc = scales[buf];
      const uint32_t off = buf * bytes_bc;
      // a tile of scores C_t . B_s (none above the diagonal), and what the state before the chunk gives, S^T C_t: eight columns
      // of S, the high parts' two pieces of k and the low parts' in one load.  The next step's operands are on their way.
      float p[2][4];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) p[nt][0] = p[nt][1] = p[nt][2] = p[nt][3] = 0.f;
      uint32_t a[2][4], bb[2][4], ss[2][4];
      auto ask = [&](int w, int k) {
        ldmatrix_x4(a[w][0], a[w][1], a[w][2], a[w][3], aC + off + k * 2);
        if (mj <= mi) ldmatrix_x4(bb[w][0], bb[w][1], bb[w][2], bb[w][3], aB + off + k * 2);
        ldmatrix_x4_trans(ss[w][0], ss[w][1], ss[w][2], ss[w][3], aS + k * (SC_PV * 2));
      };
      auto use = [&](int w) {
        if (mj <= mi) {
          mma_bf16(p[0], a[w][0], a[w][1], a[w][2], a[w][3], bb[w][0], bb[w][1]);
          mma_bf16(p[1], a[w][0], a[w][1], a[w][2], a[w][3], bb[w][2], bb[w][3]);
        }
        mma_bf16(Y, a[w][0], a[w][1], a[w][2], a[w][3], ss[w][0], ss[w][1]);
        mma_bf16(Y2, a[w][0], a[w][1], a[w][2], a[w][3], ss[w][2], ss[w][3]);
      };
      ask(0, 0);
      for (int k = 0; k < N; k += 32) {
        if (k + 16 < N) ask(1, k + 16);
        use(0);
        if (k + 32 < N) ask(0, k + 32);
        if (k + 16 < N) use(1);
      }
      // S <- 2^(L_end) S + sum_s B_s (w_s x_s)^T
      const float keep = sc.end[0];
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        if (srow + 128 * r < N) {
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) { S[r][nt][0] *= keep; S[r][nt][1] *= keep; S[r][nt][2] *= keep; S[r][nt][3] *= keep; }
#pragma unroll
          for (int k2 = 0; k2 < 2; ++k2) {
            uint32_t h[2][4];
#pragma unroll
            for (int w = 0; w < 2; ++w) {
              const int ks = 2 * k2 + w;
              ldmatrix_x4_trans(a[w][0], a[w][1], a[w][2], a[w][3], aBt + off + (ks * 16 * PN + 128 * r) * 2);
              ldmatrix_x4_trans(bb[w][0], bb[w][1], bb[w][2], bb[w][3], aW + ks * (16 * SC_PV * 2));
              ldmatrix_x4_trans(h[w][0], h[w][1], h[w][2], h[w][3], aW + to_wl + ks * (16 * SC_PV * 2));
            }
#pragma unroll
            for (int w = 0; w < 2; ++w) {
              mma_bf16(S[r][0], a[w][0], a[w][1], a[w][2], a[w][3], bb[w][0], bb[w][1]);
              mma_bf16(S[r][1], a[w][0], a[w][1], a[w][2], a[w][3], bb[w][2], bb[w][3]);
              mma_bf16(S[r][0], a[w][0], a[w][1], a[w][2], a[w][3], h[w][0], h[w][1]);
              mma_bf16(S[r][1], a[w][0], a[w][1], a[w][2], a[w][3], h[w][2], h[w][3]);
            }
          }
        }
      }
      if (mj <= mi) {
        const float La = sc.L[m0 + g], Lb = sc.L[m0 + g + 8];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const int s = mj * 16 + nt * 8 + 2 * t4, row = m0 + g;
          const float2 q = *reinterpret_cast<const float2*>(sc.q + s);
          p[nt][0] = s <= row ? p[nt][0] * fast_exp2(La - q.x) : 0.f;
          p[nt][1] = s + 1 <= row ? p[nt][1] * fast_exp2(La - q.y) : 0.f;
          p[nt][2] = s <= row + 8 ? p[nt][2] * fast_exp2(Lb - q.x) : 0.f;
          p[nt][3] = s + 1 <= row + 8 ? p[nt][3] * fast_exp2(Lb - q.y) : 0.f;
          uint32_t hi, lo;
          split2(p[nt][0], p[nt][1], hi, lo);
          *reinterpret_cast<uint32_t*>(Ph + row * SC_PP + s) = hi;
          *reinterpret_cast<uint32_t*>(Pl + row * SC_PP + s) = lo;
          split2(p[nt][2], p[nt][3], hi, lo);
          *reinterpret_cast<uint32_t*>(Ph + (row + 8) * SC_PP + s) = hi;
          *reinterpret_cast<uint32_t*>(Pl + (row + 8) * SC_PP + s) = lo;
        }
      }
      const float ea = sc.e[m0 + g], eb = sc.e[m0 + g + 8];
      Y[0] *= ea; Y[1] *= ea; Y[2] *= eb; Y[3] *= eb;
      Y2[0] *= ea; Y2[1] *= ea; Y2[2] *= eb; Y2[3] *= eb;
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();                       // (2)
    if (!worker) continue;
    // the chunk's own tokens: the weighted scores times x
#pragma unroll
    for (int k2 = 0; k2 < 2; ++k2) {
      if (2 * k2 <= mi) {
        uint32_t b0, b1, b2, b3, h[2][4], l[2][4];
        ldmatrix_x4_trans(b0, b1, b2, b3, aX + buf * bytes_x + k2 * (32 * SC_PV * 2));      // 32 tokens, eight columns
        ldmatrix_x4(h[0][0], h[0][1], h[0][2], h[0][3], aP + k2 * 64);
        ldmatrix_x4(l[0][0], l[0][1], l[0][2], l[0][3], aP + to_pl + k2 * 64);
        if (2 * k2 + 1 <= mi) {
          ldmatrix_x4(h[1][0], h[1][1], h[1][2], h[1][3], aP + k2 * 64 + 32);
          ldmatrix_x4(l[1][0], l[1][1], l[1][2], l[1][3], aP + to_pl + k2 * 64 + 32);
        }
        mma_bf16(Y, h[0][0], h[0][1], h[0][2], h[0][3], b0, b1);
        mma_bf16(Y2, l[0][0], l[0][1], l[0][2], l[0][3], b0, b1);
        if (2 * k2 + 1 <= mi) {
          mma_bf16(Y, h[1][0], h[1][1], h[1][2], h[1][3], b2, b3);
          mma_bf16(Y2, l[1][0], l[1][1], l[1][2], l[1][3], b2, b3);
        }
      }
    }
    if (more) lay_out(buf ^ 1);
    const int n = min(SC_T, t1 - c0), c = mj * 8 + 2 * t4;
    if (col0 + c < V) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = m0 + g + half * 8;
        if (row >= n) continue;
        const uint32_t v = *reinterpret_cast<const uint32_t*>(xs + (buf * SC_T + row) * SC_PV + c);
        *reinterpret_cast<float2*>(y + (size_t)(c0 + row) * z.inner() + (size_t)h * V + col0 + c) =
            make_float2(fmaf(sk, __uint_as_float(v << 16), Y[2 * half] + Y2[2 * half]),
                        fmaf(sk, __uint_as_float(v & 0xffff0000u), Y[2 * half + 1] + Y2[2 * half + 1]));
      }
    }
  }
  if (!worker) return;
  if (!write_state) return;
#pragma unroll
  for (int r = 0; r < RT; ++r)
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const int n = srow + 128 * r + g, c = nt * 8 + 2 * t4;
      if (srow + 128 * r >= N || col0 + scol + c >= V) continue;
      *reinterpret_cast<float2*>(st + (size_t)n * V + c) = make_float2(S[r][nt][0], S[r][nt][1]);
      *reinterpret_cast<float2*>(st + (size_t)(n + 8) * V + c) = make_float2(S[r][nt][2], S[r][nt][3]);
    }
}

// 1 if ssm_chunks takes the sizes: state sizes in steps of 16, value sizes in steps of 8, both up to 256
AB_API int ab_ssm_chunks_supports(int N, int V) { return N > 0 && N <= 256 && N % 16 == 0 && V > 0 && V <= 256 && V % 8 == 0 ? 1 : 0; }

// xbc bfloat16 [T, channels] (x | B | C), la and dt float32 [T, H] (log decays, step sizes), y float32 [T, H * V].
AB_API int ab_ssm_chunks(const void* xbc, const float* la, const float* dt, const float* skip, float* state, float* y,
                         const int* cu_q, const int* slots, int n_seqs, int H, int G, int N, int V, int write_state,
                         cudaStream_t stream) {
  if (n_seqs <= 0) return AB_OK;
  const SsmSizes z{H, G, N, V, 1};
  if (!ssm_sizes_ok(z) || !ab_ssm_chunks_supports(N, V) || H > 65535 || ((((uintptr_t)xbc) | ((uintptr_t)state)) & 15)) return AB_BAD_ARG;
  if ((H * V) % 8 || (G * N) % 8) return AB_BAD_ARG;              // rows of 16-byte pieces
  const dim3 grid((unsigned)n_seqs, (unsigned)H, (unsigned)((V + SC_CV - 1) / SC_CV));
  const size_t smem = chunk_smem(N);
#define AB_GO(RT)                                                                                                      \
  {                                                                                                                    \
    cudaError_t e = cudaFuncSetAttribute(ssm_chunks_kernel<RT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    if (e != cudaSuccess) return AB_CUDA_ERR + (int)e;                                                                 \
    ab_launch(ssm_chunks_kernel<RT>, grid, dim3(SC_THREADS), smem, stream, (const bf16*)xbc, la, dt, skip, state, y, cu_q, slots, \
              z, write_state);                                                                                         \
  }
  if (N <= 128) AB_GO(1) else AB_GO(2)
#undef AB_GO
  return ab_launch_status();
}

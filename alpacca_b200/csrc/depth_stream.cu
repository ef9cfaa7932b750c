// Kernels on the float32 residual stream of blocks whose sub-layers read the stream itself, whose norms act on the
// sub-layers' outputs, whose mixers see the stream through a short causal convolution and whose results are averaged
// over depth:
//
//   embed_positions  x[t] = scale * table[token_t] + pos[place_t]               token rows plus learned position rows
//   input_conv       h[t] = x[t] + sum_j w[:, j] x[t - taps + 1 + j]            per channel over time, zeros before the
//                    sequence's start; a sequence's last taps - 1 rows of x are its state, kept from step to step
//   post_norm_stream v = x[t] + y[t] / sqrt(mean(y[t]^2) + eps) * w             a sub-layer's output joins the stream;
//                    then, each if it is asked for,
//                      stores v;   dots[t] = v . g  (one number per token for a part that reads v);
//                      m = sum_(j < n) c_j X_j[t] + c_n v,  stored              the average over what earlier layers left
//                      (without it m = v)
//                      out[t] = cast(m), or, in a step of one token per sequence, cast of the next layer's
//                      input_conv of m, whose state moves on                    the next reader's input
//
// Arithmetic is 32-bit.  Rows whose sequence index is negative (padding of a captured step) leave the stream and the
// states alone.  Which thread adds what depends on the width and the launch shape alone, so a row's result does not
// depend on the rest of the batch.
#include "common.cuh"
#include "launch.cuh"

template <typename T> struct Quad;
template <> struct Quad<float> {
  __device__ __forceinline__ static float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ static void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Quad<bf16> {
  __device__ __forceinline__ static float4 load(const bf16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16),
                       __uint_as_float(v.y & 0xffff0000u));
  }
  __device__ __forceinline__ static void store(bf16* p, float4 a) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(a.x, a.y), hi = __floats2bfloat162_rn(a.z, a.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
  }
};
__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
__device__ __forceinline__ float4 axpy4(float a, float4 b, float4 c) {
  return make_float4(fmaf(a, b.x, c.x), fmaf(a, b.y, c.y), fmaf(a, b.z, c.z), fmaf(a, b.w, c.w));
}
__device__ __forceinline__ float dot4(float4 a, float4 b) { return (a.x * b.x + a.y * b.y) + (a.z * b.z + a.w * b.w); }

// ---------------------------------------------------------------------------
// embedding
// ---------------------------------------------------------------------------
template <typename T, bool VEC>
__global__ void embed_positions_kernel(const T* __restrict__ table, const T* __restrict__ pos, const int* __restrict__ tokens,
                                       const int* __restrict__ tok_seq, const int* __restrict__ tok_pos, float scale,
                                       float* __restrict__ out, int width) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  float* o = out + (size_t)t * width;
  if (tok_seq[t] < 0) {
    for (int j = threadIdx.x; j < width; j += blockDim.x) o[j] = 0.f;
    return;
  }
  const T* e = table + (size_t)tokens[t] * width;
  const T* p = pos + (size_t)tok_pos[t] * width;
  if (VEC) {
    for (int j = threadIdx.x * 4; j < width; j += blockDim.x * 4) {
      const float4 a = Quad<T>::load(e + j), b = Quad<T>::load(p + j);
      *reinterpret_cast<float4*>(o + j) = axpy4(scale, a, b);
    }
  } else {
    for (int j = threadIdx.x; j < width; j += blockDim.x) o[j] = fmaf(scale, to_f32(e[j]), to_f32(p[j]));
  }
}

AB_API int ab_embed_positions(const void* table, const void* pos, int dtype, const int* tokens, const int* tok_seq,
                              const int* tok_pos, float scale, float* out, int n_tokens, int width, cudaStream_t stream) {
  if (n_tokens <= 0 || width <= 0) return AB_OK;
  const int threads = width >= 1024 ? 256 : 128;
#define AB_GO(T, V)                                                                                                    \
  ab_launch(embed_positions_kernel<T, V>, dim3((unsigned)n_tokens), dim3(threads), 0, stream, (const T*)table, (const T*)pos, \
            tokens, tok_seq, tok_pos, scale, out, width)
  if (dtype == AB_F32) { if (width % 4 == 0) AB_GO(float, true); else AB_GO(float, false); }
  else if (dtype == AB_BF16) { if (width % 4 == 0) AB_GO(bf16, true); else AB_GO(bf16, false); }
  else return AB_BAD_ARG;
#undef AB_GO
  return ab_launch_status();
}

// ---------------------------------------------------------------------------
// input convolution
// ---------------------------------------------------------------------------
// w: [taps, width] (tap by tap); state: [slots, taps - 1, width], the oldest row first.  A block takes one token and
// NC * blockDim channels.  A token whose taps all lie in this step reads the stream alone.  The first taps - 1 tokens
// of a sequence's step also read the state: the block of the FIRST token does all of them, channel by channel, and
// then moves the state on (each thread reads the channels it writes before it writes them).
template <typename T, int NC>
__global__ void __launch_bounds__(256)
input_conv_kernel(const float* __restrict__ x, const float* __restrict__ w, float* __restrict__ state, T* __restrict__ out,
                  const int* __restrict__ tok_seq, const int* __restrict__ cu_q, const int* __restrict__ slots, int width,
                  int taps, int write_state) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * NC;
  if (c >= width) return;
  const int b = tok_seq[t];
  if (b < 0) {
#pragma unroll
    for (int e = 0; e < NC; ++e) out[(size_t)t * width + c + e] = from_f32<T>(0.f);
    return;
  }
  const int first = cu_q[b], keep = taps - 1;
  const int i = t - first;
  auto load = [&](const float* p, float (&v)[NC]) {
    if (NC == 4) {
      const float4 q = *reinterpret_cast<const float4*>(p);
      v[0] = q.x; v[NC > 1 ? 1 : 0] = q.y; v[NC > 2 ? 2 : 0] = q.z; v[NC > 3 ? 3 : 0] = q.w;
    } else {
      v[0] = *p;
    }
  };
  auto finish = [&](int tt, const float (&acc)[NC]) {
    float self[NC];
    load(x + (size_t)tt * width + c, self);
    if (NC == 4) {
      Quad<T>::store(out + (size_t)tt * width + c,
                     make_float4(self[0] + acc[0], self[NC > 1 ? 1 : 0] + acc[NC > 1 ? 1 : 0],
                                 self[NC > 2 ? 2 : 0] + acc[NC > 2 ? 2 : 0], self[NC > 3 ? 3 : 0] + acc[NC > 3 ? 3 : 0]));
    } else {
      out[(size_t)tt * width + c] = from_f32<T>(self[0] + acc[0]);
    }
  };
  if (i >= keep && i > 0) {
    float acc[NC];
#pragma unroll
    for (int e = 0; e < NC; ++e) acc[e] = 0.f;
    for (int j = 0; j < taps; ++j) {
      float v[NC], wv[NC];
      load(x + (size_t)(t - keep + j) * width + c, v);
      load(w + (size_t)j * width + c, wv);
#pragma unroll
      for (int e = 0; e < NC; ++e) acc[e] = fmaf(wv[e], v[e], acc[e]);
    }
    finish(t, acc);
    return;
  }
  if (i > 0) return;                                      // done by the block of the sequence's first token
  const int n = cu_q[b + 1] - first;
  float* st = keep > 0 ? state + (size_t)slots[b] * keep * width + c : nullptr;
  const int todo = n < (keep > 1 ? keep : 1) ? n : (keep > 1 ? keep : 1);
  for (int q = 0; q < todo; ++q) {
    float acc[NC];
#pragma unroll
    for (int e = 0; e < NC; ++e) acc[e] = 0.f;
    for (int j = 0; j < taps; ++j) {
      const int at = q - keep + j;                        // place among the step's tokens; before them: the state
      float v[NC], wv[NC];
      load(at >= 0 ? x + (size_t)(first + at) * width + c : st + (size_t)(keep + at) * width, v);
      load(w + (size_t)j * width + c, wv);
#pragma unroll
      for (int e = 0; e < NC; ++e) acc[e] = fmaf(wv[e], v[e], acc[e]);
    }
    finish(first + q, acc);
  }
  if (!write_state) return;
  for (int j = 0; j < keep; ++j) {                        // row j of the new state: place n - keep + j
    const int at = n - keep + j;
    float v[NC];
    load(at >= 0 ? x + (size_t)(first + at) * width + c : st + (size_t)(keep + at) * width, v);
#pragma unroll
    for (int e = 0; e < NC; ++e) st[(size_t)j * width + e] = v[e];
  }
}

// The same for steps of many tokens, TAPS of 2 to 4 and widths that are multiples of 4: a thread keeps its channels' taps and the last rows in
// registers and walks CONV_RUN packed tokens, so that a row is read once.  The tokens whose taps reach before the step
// are left to the block whose run holds the sequence's first token, which does them as the kernel above does.
#define CONV_RUN 8
template <typename T, int TAPS>
__global__ void __launch_bounds__(256)
input_conv_run_kernel(const float* __restrict__ x, const float* __restrict__ w, float* __restrict__ state, T* __restrict__ out,
                      const int* __restrict__ tok_seq, const int* __restrict__ cu_q, const int* __restrict__ slots,
                      int n_tokens, int width, int write_state) {
  constexpr int KEEP = TAPS - 1;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
  float4 wv[TAPS];
  if (c < width)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) wv[j] = *reinterpret_cast<const float4*>(w + (size_t)j * width + c);
  pdl_wait();
  pdl_trigger();
  if (c >= width) return;
  const int t0 = blockIdx.x * CONV_RUN, t1 = min(t0 + CONV_RUN, n_tokens);
  auto row = [&](int t) { return *reinterpret_cast<const float4*>(x + (size_t)t * width + c); };
  auto emit = [&](int t, const float4 (&prev)[KEEP], float4 cur) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) acc = fma4(wv[j], prev[j], acc);
    acc = fma4(wv[KEEP], cur, acc);
    Quad<T>::store(out + (size_t)t * width + c, make_float4(cur.x + acc.x, cur.y + acc.y, cur.z + acc.z, cur.w + acc.w));
  };
  float4 prev[KEEP];
  {
    // the usual case: a whole run inside one sequence, past its first KEEP tokens: every row is asked for at once
    const int b = tok_seq[t0];
    if (b >= 0 && t1 - t0 == CONV_RUN && tok_seq[t1 - 1] == b && t0 - cu_q[b] >= KEEP) {
      float4 r[CONV_RUN + KEEP];
#pragma unroll
      for (int j = 0; j < CONV_RUN + KEEP; ++j) r[j] = row(t0 - KEEP + j);
#pragma unroll
      for (int q = 0; q < CONV_RUN; ++q) {
#pragma unroll
        for (int j = 0; j < KEEP; ++j) prev[j] = r[q + j];
        emit(t0 + q, prev, r[q + KEEP]);
      }
      return;
    }
  }
  bool have = false;                       // prev holds the rows before token t
  for (int t = t0; t < t1; ++t) {
    const int b = tok_seq[t];
    if (b < 0) {
      Quad<T>::store(out + (size_t)t * width + c, make_float4(0.f, 0.f, 0.f, 0.f));
      have = false;
      continue;
    }
    const int first = cu_q[b];
    const int i = t - first;
    if (i >= KEEP) {
      if (!have)
#pragma unroll
        for (int j = 0; j < KEEP; ++j) prev[j] = row(t - KEEP + j);
      const float4 cur = row(t);
      emit(t, prev, cur);
#pragma unroll
      for (int j = 0; j + 1 < KEEP; ++j) prev[j] = prev[j + 1];
      prev[KEEP - 1] = cur;
      have = true;
      continue;
    }
    have = false;
    if (i > 0) continue;
    // a sequence's first token: its first KEEP tokens from the kept rows on, then the new kept rows
    const int n = cu_q[b + 1] - first;
    float* st = state + (size_t)slots[b] * KEEP * width + c;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) prev[j] = *reinterpret_cast<const float4*>(st + (size_t)j * width);
    for (int q = 0; q < KEEP && q < n; ++q) {
      const float4 cur = row(first + q);
      emit(first + q, prev, cur);
#pragma unroll
      for (int j = 0; j + 1 < KEEP; ++j) prev[j] = prev[j + 1];
      prev[KEEP - 1] = cur;
    }
    if (write_state)
#pragma unroll
      for (int j = 0; j < KEEP; ++j) {      // after fewer than KEEP tokens `prev` holds old and new rows, in order
        const float4 v = n < KEEP ? prev[j] : row(first + n - KEEP + j);
        *reinterpret_cast<float4*>(st + (size_t)j * width) = v;
      }
  }
}

AB_API int ab_input_conv(const float* x, const float* w, float* state, void* out, int dtype, const int* tok_seq,
                         const int* cu_q, const int* slots, int n_tokens, int width, int taps, int write_state,
                         cudaStream_t stream) {
  if (n_tokens <= 0 || width <= 0) return AB_OK;
  if (taps < 1 || (taps > 1 && !state)) return AB_BAD_ARG;
  const bool vec = width % 4 == 0;
  const int units = vec ? width / 4 : width;
  const int threads = units >= 256 ? 256 : (units + 31) / 32 * 32;
  const dim3 grid((unsigned)n_tokens, (unsigned)((units + threads - 1) / threads));
  if (n_tokens >= 256 && vec && taps >= 2 && taps <= 4 && (dtype == AB_F32 || dtype == AB_BF16)) {
    const dim3 runs((unsigned)((n_tokens + CONV_RUN - 1) / CONV_RUN), grid.y);
#define AB_RUN(T, TAPS)                                                                                               \
  ab_launch(input_conv_run_kernel<T, TAPS>, runs, dim3(threads), 0, stream, x, w, state, (T*)out, tok_seq, cu_q, slots, \
            n_tokens, width, write_state)
    if (dtype == AB_F32) { if (taps == 2) AB_RUN(float, 2); else if (taps == 3) AB_RUN(float, 3); else AB_RUN(float, 4); }
    else { if (taps == 2) AB_RUN(bf16, 2); else if (taps == 3) AB_RUN(bf16, 3); else AB_RUN(bf16, 4); }
#undef AB_RUN
    return ab_launch_status();
  }
#define AB_GO(T, NC)                                                                                                 \
  ab_launch(input_conv_kernel<T, NC>, grid, dim3(threads), 0, stream, x, w, state, (T*)out, tok_seq, cu_q, slots, width, taps, \
            write_state)
  if (dtype == AB_F32) { if (vec) AB_GO(float, 4); else AB_GO(float, 1); }
  else if (dtype == AB_BF16) { if (vec) AB_GO(bf16, 4); else AB_GO(bf16, 1); }
  else return AB_BAD_ARG;
#undef AB_GO
  return ab_launch_status();
}

// ---------------------------------------------------------------------------
// after a sub-layer
// ---------------------------------------------------------------------------
struct PostArgs {
  const float* x;              // [T, width] the stream before
  const void* y;               // [T, width] the sub-layer's output
  const float* w; float eps;   // the norm of y
  float* v_out;                // [T, width]: v (may be x); or null
  const float* g; float* dots; // [width], [T]; or null
  const float* hist; long long hist_stride; int n_hist;    // X_j at hist + j * hist_stride, j < n_hist
  const float* coef;           // [n_hist + 1]; null: no average
  float* avg_out;              // [T, width]: m; or null
  void* out;                   // [T, width] of the activation dtype; or null
  const float* conv_w; float* conv_state; const int* slots; int taps;   // the convolution of out; conv_w null: none
  const int* tok_seq;
  int width;
};

// sums over the block of three numbers at once; every thread gets them.  scratch: 3 * 32 floats
__device__ __forceinline__ void block_sum3(float& a, float& b, float& c, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  a = warp_sum(a); b = warp_sum(b); c = warp_sum(c);
  if (lane == 0) { scratch[warp] = a; scratch[32 + warp] = b; scratch[64 + warp] = c; }
  __syncthreads();
  a = warp_sum(lane < nwarps ? scratch[lane] : 0.f);
  b = warp_sum(lane < nwarps ? scratch[32 + lane] : 0.f);
  c = warp_sum(lane < nwarps ? scratch[64 + lane] : 0.f);
}

// A block per row, the row in registers: RV x 4 numbers per thread (widths that are multiples of 4).  What earlier
// layers left (the history, the convolution's kept rows) was written at least two kernels ago: it is asked for before
// the wait for the kernel before this one.
template <typename TY, typename TO, int RV, bool CONV>
__global__ void __launch_bounds__(512)
post_norm_stream_reg_kernel(const PostArgs a) {
  __shared__ float scratch[96];
  const int t = blockIdx.x, width = a.width;
  const size_t row = (size_t)t * width;
  const int b = a.tok_seq[t];
  if (b < 0) {
    pdl_wait();
    pdl_trigger();
    if (a.out != nullptr)
      for (int j = threadIdx.x; j < width; j += blockDim.x) reinterpret_cast<TO*>(a.out)[row + j] = from_f32<TO>(0.f);
    return;
  }
  float4 wv[RV], gv[RV], avg[RV];
#pragma unroll
  for (int j = 0; j < RV; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    avg[j] = gv[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i < width) {
      wv[j] = *reinterpret_cast<const float4*>(a.w + i);
      if (a.g != nullptr) gv[j] = *reinterpret_cast<const float4*>(a.g + i);
    }
  }
  float c_last = 1.f;
  if (a.coef != nullptr) {
    const float* h = a.hist + row;
#pragma unroll 4
    for (int k = 0; k < a.n_hist; ++k) {
      const float c = a.coef[k];
#pragma unroll
      for (int j = 0; j < RV; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        if (i < width) avg[j] = axpy4(c, *reinterpret_cast<const float4*>(h + (size_t)k * a.hist_stride + i), avg[j]);
      }
    }
    c_last = a.coef[a.n_hist];
  }
  // the next convolution's kept rows (up to three of them; a longer convolution fetches its rows one after another below)
  const int keep = a.taps - 1;
  float* st = CONV && keep > 0 ? a.conv_state + (size_t)a.slots[b] * keep * width : nullptr;
  constexpr int EARLY = CONV && RV <= 2 ? 3 : 0;
  const bool early = CONV && keep <= EARLY;
  float4 kept[EARLY > 0 ? EARLY : 1][RV];
  if (early) {
#pragma unroll
    for (int k = 0; k < EARLY; ++k)
#pragma unroll
      for (int j = 0; j < RV; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        if (k < keep && i < width) kept[k][j] = *reinterpret_cast<const float4*>(st + (size_t)k * width + i);
      }
  }
  pdl_wait();
  pdl_trigger();
  float4 yv[RV], xv[RV];
  float ss = 0.f, xg = 0.f, yg = 0.f;
#pragma unroll
  for (int j = 0; j < RV; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i < width) {
      yv[j] = Quad<TY>::load(reinterpret_cast<const TY*>(a.y) + row + i);
      xv[j] = *reinterpret_cast<const float4*>(a.x + row + i);
    }
  }
#pragma unroll
  for (int j = 0; j < RV; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i < width) {
      ss += dot4(yv[j], yv[j]);
      yv[j] = make_float4(yv[j].x * wv[j].x, yv[j].y * wv[j].y, yv[j].z * wv[j].z, yv[j].w * wv[j].w);
      xg += dot4(xv[j], gv[j]);
      yg += dot4(yv[j], gv[j]);
    }
  }
  block_sum3(ss, xg, yg, scratch);
  const float inv = 1.0f / sqrtf(ss / (float)width + a.eps);
  if (a.dots != nullptr && threadIdx.x == 0) a.dots[t] = fmaf(inv, yg, xg);
#pragma unroll
  for (int j = 0; j < RV; ++j) {
    const int i = (threadIdx.x + j * blockDim.x) * 4;
    if (i >= width) continue;
    float4 v = axpy4(inv, yv[j], xv[j]);
    if (a.v_out != nullptr) *reinterpret_cast<float4*>(a.v_out + row + i) = v;
    if (a.coef != nullptr) {
      v = axpy4(c_last, v, avg[j]);
      *reinterpret_cast<float4*>(a.avg_out + row + i) = v;
    }
    if (a.out == nullptr) continue;
    if (CONV) {
      // the next layer's convolution: the kept rows, then this one; the kept rows move up by one
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      if (early) {
#pragma unroll
        for (int k = 0; k < EARLY; ++k)
          if (k < keep) {
            acc = fma4(*reinterpret_cast<const float4*>(a.conv_w + (size_t)k * width + i), kept[k][j], acc);
            if (k > 0) *reinterpret_cast<float4*>(st + (size_t)(k - 1) * width + i) = kept[k][j];
          }
      }
      for (int k = early ? keep : 0; k < keep; ++k) {
        const float4 s = *reinterpret_cast<const float4*>(st + (size_t)k * width + i);
        acc = fma4(*reinterpret_cast<const float4*>(a.conv_w + (size_t)k * width + i), s, acc);
        if (k > 0) *reinterpret_cast<float4*>(st + (size_t)(k - 1) * width + i) = s;
      }
      acc = fma4(*reinterpret_cast<const float4*>(a.conv_w + (size_t)keep * width + i), v, acc);
      if (keep > 0) *reinterpret_cast<float4*>(st + (size_t)(keep - 1) * width + i) = v;
      v = make_float4(v.x + acc.x, v.y + acc.y, v.z + acc.z, v.w + acc.w);
    }
    Quad<TO>::store(reinterpret_cast<TO*>(a.out) + row + i, v);
  }
}

// The same for any width, one number at a time; a thread meets its own elements again, so nothing is kept.
template <typename TY, typename TO>
__global__ void __launch_bounds__(256)
post_norm_stream_kernel(const PostArgs a) {
  __shared__ float scratch[96];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x, width = a.width;
  const size_t row = (size_t)t * width;
  const int b = a.tok_seq[t];
  if (b < 0) {
    if (a.out != nullptr)
      for (int j = threadIdx.x; j < width; j += blockDim.x) reinterpret_cast<TO*>(a.out)[row + j] = from_f32<TO>(0.f);
    return;
  }
  const TY* y = reinterpret_cast<const TY*>(a.y) + row;
  float ss = 0.f, xg = 0.f, yg = 0.f;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float v = to_f32(y[i]);
    ss += v * v;
    if (a.g != nullptr) {
      xg += a.x[row + i] * a.g[i];
      yg += v * a.w[i] * a.g[i];
    }
  }
  block_sum3(ss, xg, yg, scratch);
  const float inv = 1.0f / sqrtf(ss / (float)width + a.eps);
  if (a.dots != nullptr && threadIdx.x == 0) a.dots[t] = fmaf(inv, yg, xg);
  const int keep = a.taps - 1;
  float* st = a.conv_w != nullptr && keep > 0 ? a.conv_state + (size_t)a.slots[b] * keep * width : nullptr;
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    float v = fmaf(inv, to_f32(y[i]) * a.w[i], a.x[row + i]);
    if (a.v_out != nullptr) a.v_out[row + i] = v;
    if (a.coef != nullptr) {
      float m = 0.f;
      for (int k = 0; k < a.n_hist; ++k) m = fmaf(a.coef[k], a.hist[(size_t)k * a.hist_stride + row + i], m);
      v = fmaf(a.coef[a.n_hist], v, m);
      a.avg_out[row + i] = v;
    }
    if (a.out == nullptr) continue;
    if (a.conv_w != nullptr) {
      float acc = 0.f;
      for (int k = 0; k < keep; ++k) {
        const float s = st[(size_t)k * width + i];
        acc = fmaf(a.conv_w[(size_t)k * width + i], s, acc);
        if (k > 0) st[(size_t)(k - 1) * width + i] = s;
      }
      acc = fmaf(a.conv_w[(size_t)keep * width + i], v, acc);
      if (keep > 0) st[(size_t)(keep - 1) * width + i] = v;
      v += acc;
    }
    reinterpret_cast<TO*>(a.out)[row + i] = from_f32<TO>(v);
  }
}

AB_API int ab_post_norm_stream(const float* x, const void* y, int y_dtype, const float* w, float eps, float* v_out,
                               const float* g, float* dots, const float* hist, long long hist_stride, int n_hist,
                               const float* coef, float* avg_out, void* out, int out_dtype, const float* conv_w,
                               float* conv_state, const int* slots, int taps, const int* tok_seq, int n_rows, int width,
                               cudaStream_t stream) {
  if (n_rows <= 0 || width <= 0) return AB_OK;
  if (!x || !y || !w || !tok_seq || (dots && !g) || (coef && (!avg_out || n_hist < 0 || (n_hist > 0 && !hist)))) return AB_BAD_ARG;
  if (conv_w && (!out || taps < 1 || (taps > 1 && (!conv_state || !slots)))) return AB_BAD_ARG;
  if ((y_dtype != AB_F32 && y_dtype != AB_BF16) || (out && out_dtype != AB_F32 && out_dtype != AB_BF16)) return AB_BAD_ARG;
  PostArgs a{x, y, w, eps, v_out, g, dots, hist, hist_stride, n_hist, coef, avg_out, out, conv_w, conv_state, slots,
             conv_w ? taps : 1, tok_seq, width};
  const bool of = !out || out_dtype == AB_F32;
  const int threads = width >= 4096 ? 512 : (width >= 1024 ? 256 : 128);
  const int rv = width % 4 == 0 ? (width / 4 + threads - 1) / threads : 99;
#define AB_REG(TY, TO, RV)                                                                                              \
  {                                                                                                                     \
    if (conv_w != nullptr)                                                                                              \
      ab_launch(post_norm_stream_reg_kernel<TY, TO, RV, true>, dim3((unsigned)n_rows), dim3(threads), 0, stream, a);    \
    else                                                                                                                \
      ab_launch(post_norm_stream_reg_kernel<TY, TO, RV, false>, dim3((unsigned)n_rows), dim3(threads), 0, stream, a);   \
  }
#define AB_GO(TY, TO)                                                                                            \
  {                                                                                                              \
    if (rv <= 1) AB_REG(TY, TO, 1)                                                                               \
    else if (rv <= 2) AB_REG(TY, TO, 2)                                                                          \
    else if (rv <= 4) AB_REG(TY, TO, 4)                                                                          \
    else ab_launch(post_norm_stream_kernel<TY, TO>, dim3((unsigned)n_rows), dim3(256), 0, stream, a);            \
  }
  if (y_dtype == AB_F32) { if (of) AB_GO(float, float) else AB_GO(float, bf16) }
  else { if (of) AB_GO(bf16, float) else AB_GO(bf16, bf16) }
#undef AB_GO
#undef AB_REG
  return ab_launch_status();
}

// Which experts a token has and with which weights, and the experts' activations: shared by the kernels of routed experts.
#pragma once
#include "common.cuh"

// The choice comes from a router (idx, wts), or from the token's id: row token_t of a table names its experts, each with
// the same constant weight.
struct Choice {
  const int* idx; const float* wts;       // [T, top], from a router
  const int* table; const int* tokens;    // [vocab, top], [T]: by token id (idx null)
  float weight;                           // of every expert chosen by table
};
__device__ __forceinline__ int chosen_expert(const Choice& c, int t, int k, int top) {
  return c.idx != nullptr ? c.idx[(size_t)t * top + k] : c.table[(size_t)c.tokens[t] * top + k];
}
__device__ __forceinline__ float chosen_weight(const Choice& c, int t, int k, int top) {
  return c.idx != nullptr ? c.wts[(size_t)t * top + k] : c.weight;
}
static inline bool choice_ok(const Choice& c) { return c.idx ? c.wts != nullptr : (c.table != nullptr && c.tokens != nullptr); }

__device__ __forceinline__ float gelu_erf(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752440f)); }
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
#define MOE_ACT_KINDS 3      // 0 GELU (erf), 1 SiLU, 2 the square of ReLU
__device__ __forceinline__ float activate(float z, int kind) {
  if (kind == 2) {
    const float r = fmaxf(z, 0.f);
    return r * r;
  }
  return kind == 0 ? gelu_erf(z) : silu(z);
}
// An expert's inner value from its products g (gate; unused without one) and u with the token's row: the weight w of a
// chosen expert multiplies the expert's input (`weight_in`; both products are linear in it) or the inner value.
template <bool GATED>
__device__ __forceinline__ float expert_inner(float g, float u, float w, int weight_in, int kind) {
  const float in = weight_in ? w : 1.0f, after = weight_in ? 1.0f : w;
  return GATED ? after * activate(in * g, kind) * (in * u) : after * activate(in * u, kind);
}

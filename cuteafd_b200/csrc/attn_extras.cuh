// What a grouped-query attention layer may have besides scores and values, shared by the decode, prefill and ordinary-core kernels and the
// merge of split partials: the first keys of the sequence staying visible behind a sliding window, a sink logit per head, a sigmoid gate on
// the output (one per head, or one per output value) and a constant factor.
#pragma once
#include "stack_rows.cuh"

template <typename T>
struct AttnExtras {
  const float* sink;        // [Hq], or null
  const T* gate;            // gate logits, rows ldg apart: column h (per head) or column h * dv + i (per value); null = none
  int ldg, gate_values, keep_first;
  float out_scale;
  // Tiles of `tile` keys that hold kept keys and lie wholly in front of the window's first tile.
  __device__ __forceinline__ int kept_tiles(int first_tile, int tile) const { return min((keep_first + tile - 1) / tile, first_tile); }
  __device__ __forceinline__ float head_factor(int t, int h) const {
    return gate && !gate_values ? out_scale / (1.f + expf(-to_f(gate[(size_t)t * ldg + h]))) : out_scale;
  }
  __device__ __forceinline__ float value_factor(int t, int col) const {
    return gate && gate_values ? 1.f / (1.f + expf(-to_f(gate[(size_t)t * ldg + col]))) : 1.f;
  }
};

struct CaAttnExtras { const float* sink; const void* gate; int ldg, gate_values, keep_first; float out_scale; };

// Without a window every key is visible: there is nothing to keep.
template <typename T>
static inline AttnExtras<T> attn_extras(const CaAttnExtras* e, int window) {
  if (!e) return AttnExtras<T>{nullptr, nullptr, 0, 0, 0, 1.f};
  return AttnExtras<T>{e->sink, (const T*)e->gate, e->ldg, e->gate_values, window > 0 && e->keep_first > 0 ? e->keep_first : 0, e->out_scale};
}

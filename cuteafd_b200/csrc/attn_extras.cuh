// What a grouped-query attention layer may have besides scores and values, shared by the decode, prefill and ordinary-core kernels and the
// merge of split partials: the first keys of the sequence staying visible behind a sliding window, or one mean key and value for each block of
// tokens that lies wholly in front of it; a sink logit per head, a sigmoid gate on the output (one per head, or one per output value) and a
// constant factor.
//
// Pooled blocks: block b holds the positions [b P, b P + P).  Its row (laid out like the token rows) is kept in strips of eight blocks, and a strip
// belongs to the page of its first token: strip s to page s P / 8, as the (s - ceil(8 j / P))-th strip of logical page j.  So pooled rows
// need no pages of their own, are freed and used again with the tokens' pages, and eight of them are one 1 KB box of a 64-wide chunk whatever P is.
#pragma once
#include "stack_rows.cuh"

template <typename T>
struct AttnExtras {
  const float* sink;        // [Hq], or null
  const T* gate;            // gate logits, rows ldg apart: column h (per head) or column h * dv + i (per value); null = none
  int ldg, gate_values, keep_first;
  float out_scale;
  const T* pooled; const CUtensorMap* pool_maps;            // pooled rows of the layer, and their key and value descriptors (boxes of eight rows)
  int pool, pool_rows;                                      // tokens of a block (0: none), rows of blocks per page
  // Blocks that position `pos` sees: those whose last token lies in front of its window.
  __device__ __forceinline__ int blocks_seen(int pos, int window) const { return pool > 0 && pos >= window ? (pos - window + 1) / pool : 0; }
  // First pooled row of strip s.
  __device__ __forceinline__ int strip_row(int s, const int* table) const {
    const int j = (int)(((long long)s * pool) >> 3);
    return table[j] * pool_rows + (s - (8 * j + pool - 1) / pool) * 8;
  }
  // Tiles in front of the window's: pooled blocks, or kept keys.
  __device__ __forceinline__ int lead_tiles(int first_tile, int tile, int last_pos, int window) const {
    return pool > 0 ? (blocks_seen(last_pos, window) + tile - 1) / tile : kept_tiles(first_tile, tile);
  }
  // Tiles of `tile` keys that hold kept keys and lie wholly in front of the window's first tile.
  __device__ __forceinline__ int kept_tiles(int first_tile, int tile) const { return min((keep_first + tile - 1) / tile, first_tile); }
  __device__ __forceinline__ float head_factor(int t, int h) const {
    return gate && !gate_values ? out_scale / (1.f + expf(-to_f(gate[(size_t)t * ldg + h]))) : out_scale;
  }
  __device__ __forceinline__ float value_factor(int t, int col) const {
    return gate && gate_values ? 1.f / (1.f + expf(-to_f(gate[(size_t)t * ldg + col]))) : 1.f;
  }
};

struct CaAttnExtras { const float* sink; const void* gate; const void* pooled; const void* pool_maps; int ldg, gate_values, keep_first, pool, pool_rows; float out_scale; };

// Kept keys and pooled blocks exclude each other.
static inline bool attn_extras_ok(const CaAttnExtras* e, bool maps) {
  return !e || e->pool == 0 || (e->pool > 0 && e->pool_rows == (8 + e->pool - 1) / e->pool * 8 && (maps ? e->pool_maps : e->pooled) && !e->keep_first);
}
// Without a window every key is visible: there is nothing to keep or to pool.
template <typename T>
static inline AttnExtras<T> attn_extras(const CaAttnExtras* e, int window) {
  if (!e) return AttnExtras<T>{nullptr, nullptr, 0, 0, 0, 1.f, nullptr, nullptr, 0, 0};
  return AttnExtras<T>{e->sink, (const T*)e->gate, e->ldg, e->gate_values, window > 0 && e->keep_first > 0 ? e->keep_first : 0, e->out_scale,
                       (const T*)e->pooled, (const CUtensorMap*)e->pool_maps, window > 0 ? e->pool : 0, e->pool_rows};
}

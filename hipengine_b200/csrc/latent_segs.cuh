// Portions of several requests in one latent-attention launch: which keys a portion sees and where they lie.
//
// Segment s owns rows [seg_start[s], seg_start[s+1]) of the batch, at consecutive positions from pos[seg_start[s]].  It sees
// the keys [lo, last position], lo = 0 or (with a window) the oldest key of its first row.  Gathered rows of the segments lie
// one after the other, each segment padded to a multiple of eight rows (zeros), so that 16-bit columns indexed by key start
// on 16-byte boundaries.
#pragma once
#include "common.cuh"

namespace he {

constexpr int LATENT_SEG_ALIGN = 8;

struct LatentSeg {
  int row0, T, pos0;     // first row, rows, position of the first row
  int lo, keys;          // first visible key, visible keys
  int key0;              // gathered row of key `lo`
};

__device__ __forceinline__ LatentSeg latent_seg(const int* seg_start, const int* pos, int s, int window, int key0) {
  LatentSeg g;
  g.row0 = seg_start[s];
  g.T = seg_start[s + 1] - g.row0;
  g.pos0 = pos[g.row0];
  g.lo = window > 0 ? max(0, g.pos0 - window + 1) : 0;
  g.keys = g.pos0 + g.T - g.lo;
  g.key0 = key0;
  return g;
}
__device__ __forceinline__ int latent_seg_rows(const LatentSeg& g) {
  return (g.keys + LATENT_SEG_ALIGN - 1) / LATENT_SEG_ALIGN * LATENT_SEG_ALIGN;
}

// Segment and tile of the `t`-th tile of BM rows; false past the last one.
template <int BM>
__device__ __forceinline__ bool latent_find_tile(const int* seg_start, const int* pos, int n_seg, int window, int t,
                                                 LatentSeg& g, int& tile) {
  int key0 = 0;
  for (int s = 0; s < n_seg; ++s) {
    g = latent_seg(seg_start, pos, s, window, key0);
    const int tiles = (g.T + BM - 1) / BM;
    if (t < tiles) {
      tile = t;
      return true;
    }
    t -= tiles;
    key0 += latent_seg_rows(g);
  }
  return false;
}

struct LatentPrefillArgs {
  const __nv_bfloat16* q;      // [rows][H][qd], rotated: [dn | rotated, zero-padded]
  const __nv_bfloat16* kx;     // [keys][n_heads * dn] expanded keys
  const __nv_bfloat16* v;      // [keys][n_heads * dv] expanded values, or transposed [n_heads * dv][keys] (tensor-memory form)
  const __nv_bfloat16* lat;    // [keys][W], rotated key part from column rank_cols
  const float* sink;           // [H] or null
  const int* seg_start;        // [n_seg + 1] absolute rows of q / out
  const int* pos;              // [rows]
  __nv_bfloat16* out;          // [rows][H * dv]
  int* status;
  int n_seg, tiles, H, head0, n_heads, dn, dv, qd, W, rank_cols, window;
  int rows, keys;              // rows of q / out, gathered rows
  float scale;
};

}  // namespace he

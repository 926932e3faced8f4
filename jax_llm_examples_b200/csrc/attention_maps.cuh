// What the attention kernels share beyond the plain causal window: key tiles of a window that keeps the sequence's first
// keys, and the difference of two attention maps per head.
//
// Kept first keys.  A query at position p sees key j <= p when j >= lo(p) (its window's first key) or j < keep.  A block's
// walk over key tiles then has two stretches: tiles [0, n_kept) over the kept keys below the window's first tile, then
// the window's tiles from `begin` on (a multiple of the tile size, so that the stretches never overlap).
//
// Two maps per head ("differential" attention).  Query heads 2h and 2h + 1 are the two maps of head h over the same
// values; a cached key row holds both maps' keys side by side, [map 1 | map 2 | zeros], and a map's query row is zero
// outside its own part, so that the score of a whole row against a whole row is the map's score.  With a1, a2 the
// maps' outputs, o = a1 - weight * a2 and the head's output is o / sqrt(mean(o^2) + eps) * mult over its out_dim values.
#pragma once

struct MapDifference {
  int map_dim;      // entries of one map's key
  int out_dim;      // values per head
  float weight, mult, eps;
  int pad_;
  long long ld_out; // elements between two tokens' output rows: out[n * ld_out + head * out_dim + c]
};

// Key tiles of height T that hold the kept keys below `begin`.
__host__ __device__ __forceinline__ int kept_tiles(int keep, int begin, int T) {
  const int kept = keep < begin ? keep : begin;
  return kept > 0 ? (kept + T - 1) / T : 0;
}
// First key of the walk's tile t.
__host__ __device__ __forceinline__ int walk_key(int t, int n_kept, int begin, int T) {
  return t < n_kept ? t * T : begin + (t - n_kept) * T;
}

// Which cached keys a decode step's query sees.
#pragma once
#include <cuda_runtime.h>

namespace dewb {

// First key seen by the query at position len - 1 of a row: the last `window` keys (0: all), and none from before the start of the
// query's chunk of `chunk` positions, counted from the row's first token (0: no chunks).
__device__ __forceinline__ int first_key(int len, int window, int chunk) {
  int first = (window > 0 && len > window) ? len - window : 0;
  if (chunk > 0 && len > 0) first = max(first, (len - 1) / chunk * chunk);
  return first;
}

// The same row when its first `keep` keys stay visible beside the window: the keys [0, kept) and [first, len).
__device__ __forceinline__ int kept_keys(int first, int keep) { return keep < first ? keep : first; }

// The tiles of `tk` keys that hold those keys: `kept` tiles from the row's start, then the tiles from `lo` on; each once.
struct TileWalk {
  int first, kept, lo, n;
  __device__ __forceinline__ TileWalk(int len, int window, int keep, int chunk, int tk) {
    first = first_key(len, window, chunk);
    lo = first / tk;
    kept = min((kept_keys(first, keep) + tk - 1) / tk, lo);
    n = kept + max(0, (len + tk - 1) / tk - lo);
  }
  __device__ __forceinline__ int tile(int i) const { return i < kept ? i : lo + i - kept; }
};

}  // namespace dewb

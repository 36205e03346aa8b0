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

}  // namespace dewb

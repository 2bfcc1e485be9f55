// Visibility of sliding-window attention with kept first tokens: position i sees j <= i if i - j < window or j < keep_first;
// window 0: every j <= i. The visible keys are two ranges, [0, kept) and [first, i], that do not overlap.
#pragma once
#include "common.cuh"

struct WindowRange {
  int kept, first;
};

__host__ __device__ __forceinline__ WindowRange window_range(int i, int window, int keep_first) {
  const int first = window > 0 && i >= window ? i - window + 1 : 0;
  return {keep_first < first ? keep_first : first, first};
}

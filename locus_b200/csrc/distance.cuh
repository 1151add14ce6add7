// A linear distance bias: slope[h] * (p - t) is taken off the scaled score of a query at position p with a key at position t,
// a slope per query head (`slopes` [heads] float32 in natural units, or null: no bias).  Kernels whose scores are in base 2
// use slope_log2().  The distance enters as p - t itself (not split into a part of the row and a part of the key), so that
// the form also holds beside a sink, and nothing large cancels.
#pragma once

__device__ __forceinline__ float slope_of(const float* __restrict__ slopes, int h) { return slopes ? slopes[h] : 0.f; }
__device__ __forceinline__ float slope_log2(const float* __restrict__ slopes, int h) { return slope_of(slopes, h) * 1.4426950408889634f; }

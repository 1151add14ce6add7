// Which keys a query sees, besides a window's kept first tokens: those from first_key() up to the query itself.
//   window > 0    the last `window` positions
//   chunk > 0     the positions of the query's own chunk of that many, counted from the sequence's position 0
//   neither       all of them
// (never both: refused on the host).  first_key() does not decrease with the position, so a tile of queries needs the
// keys from its first query's first key on, and a tile of keys at or behind its last query's first key is hidden from none.
#pragma once

__device__ __forceinline__ int first_key(int window, int chunk, int p) {
    if (chunk > 0) return p - p % chunk;
    return window > 0 ? max(0, p - window + 1) : 0;
}

static inline bool mask_ok(int window, int chunk, int keep_first) {
    return window >= 0 && chunk >= 0 && keep_first >= 0 && (window == 0 || chunk == 0);
}

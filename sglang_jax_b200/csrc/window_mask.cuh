// Which keys a query sees under a sliding window that keeps a sequence's first tokens, and which tiles hold them.
#pragma once

namespace sglb {

// Query at position `pos` sees key j iff j <= pos and (pos - j < size or j < keep); size 0: every key up to its own.
struct Window {
  int size, keep;
  __device__ __forceinline__ int first(int pos) const { return size > 0 && pos >= size ? pos - size + 1 : 0; }
  __device__ __forceinline__ bool sees(int pos, int j) const { return j <= pos && (j >= first(pos) || j < keep); }
};

// The tiles of `TILE` keys that queries with positions lo .. hi need, in order: those of the kept tokens, then those from
// the window of `lo` to `hi`.
template <int TILE>
struct KeyTiles {
  int kept, begin, count;                // kept tiles in front, first tile of the window, all tiles
  __device__ __forceinline__ KeyTiles(const Window& w, int lo, int hi) {
    begin = w.first(lo) / TILE;
    const int k = (w.keep + TILE - 1) / TILE;
    kept = k < begin ? k : begin;
    count = kept + hi / TILE + 1 - begin;
  }
  __device__ __forceinline__ int tile(int i) const { return i < kept ? i : begin + (i - kept); }
};

}  // namespace sglb

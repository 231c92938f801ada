// Rows and recurrent state of one sequence in a batch of portions of prompts and single decoded tokens.
#pragma once
#include <cuda_runtime.h>

namespace eredu {

struct RaggedBatch {
  const int* block_table;      // [B, max_pages]; the first page names the sequence
  const int* page_to_slot;     // [pages]: first page -> recurrent-state slot; null where nothing is kept (slot 0)
  const int* cu_q;             // [B + 1] row offsets, or null: q_per_seq rows each
  const long long* slots;      // [M] cache slots; a sequence whose first row has none (< 0) keeps its state
  int B, q_per_seq, max_pages;
};

struct RaggedSeq {
  int row0, rows, slot;
  bool live;
};

__device__ __forceinline__ RaggedSeq ragged_seq(const RaggedBatch& r, int b) {
  RaggedSeq s;
  s.row0 = r.cu_q != nullptr ? r.cu_q[b] : b * r.q_per_seq;
  s.rows = r.cu_q != nullptr ? r.cu_q[b + 1] - s.row0 : r.q_per_seq;
  s.live = s.rows > 0 && r.slots[s.row0] >= 0;
  s.slot = s.live && r.page_to_slot != nullptr ? r.page_to_slot[r.block_table[static_cast<size_t>(b) * r.max_pages]] : 0;
  return s;
}

}  // namespace eredu

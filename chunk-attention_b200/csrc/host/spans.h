// SpanBatch — the tokens of one step as the kernels read them: the next portion of each of several sequences, laid
// end to end, with positions, state slots and the piece list (ca_spans).  One pinned buffer, one upload.
#pragma once
#include <torch/torch.h>

#include <vector>

#include "../../../include/chunk_attn_b200.h"

namespace ca_host {

class SpanBatch {
  public:
    // tokens[e]: the entry's tokens; starts[e]: position of its first one; slots[e]: row of the state arrays
    SpanBatch(const std::vector<std::vector<int>>& tokens, const std::vector<int>& starts, const std::vector<int>& slots,
              torch::Device device, int work_len);
    const ca_spans* view() const { return &spans_; }

    int n_entries() const { return spans_.n_entries; }
    int n_tokens() const { return spans_.n_tokens; }
    bool single() const { return spans_.max_tokens == 1; }  // one token per entry: a decode step
    torch::Tensor tokens, positions, entry_of, last;        // int32 views of the uploaded buffer; last: row of each entry's last token
    torch::Device device() const { return buffer_.device(); }
    int max_slot() const { return max_slot_; }
    int min_token() const { return min_token_; }
    int max_token() const { return max_token_; }

  private:
    torch::Tensor buffer_;
    ca_spans spans_{};
    int max_slot_ = -1, min_token_ = 0, max_token_ = 0;
};

}  // namespace ca_host

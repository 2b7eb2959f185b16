#include "spans.h"

#include <c10/cuda/CUDAGuard.h>

#include <algorithm>
#include <cstring>
#include <stdexcept>

namespace ca_host {

SpanBatch::SpanBatch(const std::vector<std::vector<int>>& toks, const std::vector<int>& starts, const std::vector<int>& slots,
                     torch::Device device, int work_len) {
    const size_t E = toks.size();
    if (E == 0 || starts.size() != E || slots.size() != E) throw std::runtime_error("SpanBatch: one start and one slot per entry are required");
    if (work_len < 1) throw std::runtime_error("SpanBatch: work_len must be positive");
    int64_t T = 0, W = 0;
    int longest = 0;
    for (size_t e = 0; e < E; e++) {
        const int n = (int)toks[e].size();
        if (n == 0) throw std::runtime_error("SpanBatch: an entry has no tokens");
        if (starts[e] < 0 || slots[e] < 0) throw std::runtime_error("SpanBatch: negative start or slot");
        T += n;
        W += (n + work_len - 1) / work_len;
        longest = std::max(longest, n);
        max_slot_ = std::max(max_slot_, slots[e]);
    }
    std::vector<int> sorted(slots);
    std::sort(sorted.begin(), sorted.end());
    if (std::adjacent_find(sorted.begin(), sorted.end()) != sorted.end()) throw std::runtime_error("SpanBatch: two entries share a state slot");
    if (W > 65535) throw std::runtime_error("SpanBatch: too many pieces for one step");
    // work first: it is read 16 bytes at a time
    const int64_t o_work = 0, o_tok = 4 * W, o_pos = o_tok + T, o_ent = o_pos + T, o_cu = o_ent + T, o_start = o_cu + (int64_t)E + 1,
                  o_slot = o_start + (int64_t)E, o_off = o_slot + (int64_t)E, o_last = o_off + (int64_t)E + 1, total = o_last + (int64_t)E;
    torch::Tensor host = torch::empty({total}, torch::TensorOptions().dtype(torch::kInt32).pinned_memory(device.is_cuda()));
    int32_t* d = host.data_ptr<int32_t>();
    int32_t t = 0, w = 0;
    for (size_t e = 0; e < E; e++) {
        const int n = (int)toks[e].size();
        d[o_cu + e] = t;
        d[o_start + e] = starts[e];
        d[o_slot + e] = slots[e];
        d[o_off + e] = w;
        d[o_last + e] = t + n - 1;
        for (int b = 0, k = 0; b < n; b += work_len, k++, w++) {
            int32_t* q = d + o_work + 4 * (int64_t)w;
            q[0] = (int32_t)e;
            q[1] = t + b;
            q[2] = t + std::min(n, b + work_len);
            q[3] = k;
        }
        for (int i = 0; i < n; i++) {
            d[o_tok + t + i] = toks[e][i];
            min_token_ = std::min(min_token_, toks[e][i]);
            max_token_ = std::max(max_token_, toks[e][i]);
            d[o_pos + t + i] = starts[e] + i;
            d[o_ent + t + i] = (int32_t)e;
        }
        t += n;
    }
    d[o_cu + E] = t;
    d[o_off + E] = w;
    if (device.is_cuda()) {
        c10::cuda::CUDAGuard guard(device);
        buffer_ = host.to(device, torch::kInt32, /*non_blocking=*/true);
    } else {
        buffer_ = host;
    }
    const int32_t* p = buffer_.data_ptr<int32_t>();
    spans_.n_entries = (int32_t)E;
    spans_.n_tokens = (int32_t)T;
    spans_.max_tokens = longest;
    spans_.n_work = (int32_t)W;
    spans_.work_len = work_len;
    spans_.cu = p + o_cu;
    spans_.start = p + o_start;
    spans_.slot = p + o_slot;
    spans_.entry_of = p + o_ent;
    spans_.work = p + o_work;
    spans_.work_off = p + o_off;
    tokens = buffer_.narrow(0, o_tok, T);
    positions = buffer_.narrow(0, o_pos, T);
    entry_of = buffer_.narrow(0, o_ent, T);
    last = buffer_.narrow(0, o_last, (int64_t)E);
}

}  // namespace ca_host

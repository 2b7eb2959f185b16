#include "attention.h"

#include <algorithm>
#include <chrono>

#include <c10/cuda/CUDAGuard.h>
#include <c10/cuda/CUDAStream.h>

#include <cstring>
#include <iostream>
#include <stdexcept>

namespace ca_host {
namespace {

void check_rc(int rc, const char* what) {
    if (rc != CA_OK) throw std::runtime_error(std::string(what) + ": " + ca_last_error());
}

}  // namespace

Attention::Attention(int n_heads, int d_head, int chunk_size, int memory_mb, bool share_prefix, int tpp_threshold,
                     torch::Dtype dtype, torch::Device device)
  : n_heads_(n_heads), d_head_(d_head), chunk_size_(chunk_size), memory_mb_(memory_mb),
    tpp_threshold_(tpp_threshold), share_prefix_(share_prefix),
    options_(torch::TensorOptions().dtype(dtype).layout(torch::kStrided).device(device).requires_grad(false)) {
    init();
}

Attention::Attention(Attention& other)
  : n_heads_(other.n_heads_), d_head_(other.d_head_), chunk_size_(other.chunk_size_), memory_mb_(other.memory_mb_),
    tpp_threshold_(other.tpp_threshold_), shaped_(other.shaped_), shape_(other.shape_), share_prefix_(other.share_prefix_),
    options_(other.options_) {
    init();
    shared_plan_ = other.shared_plan_;  // same configuration, same sequence of tree operations: same work lists
    shared_tables_ = other.shared_tables_;
}

Attention::Attention(Attention& source, int n_heads, double scale, int window, Attention* sibling)
  : n_heads_(n_heads), d_head_(source.d_head_), chunk_size_(source.chunk_size_), memory_mb_(source.memory_mb_),
    tpp_threshold_(source.tpp_threshold_), shaped_(true), shape_(source.shape_), share_prefix_(source.share_prefix_),
    options_(source.options_) {
    source.need_latent("reader");
    if (n_heads <= 0 || window < 0) throw std::runtime_error("reader: n_heads must be positive, window not negative");
    shape_.n_heads = n_heads;
    shape_.scale = (float)scale;
    shape_.window = window;
    reader_ = true;
    pool_ = source.pool_;
    tree_ = source.tree_;
    tables_ = source.tables_;
    init();
    shared_tables_ = source.shared_tables_;
    if (sibling) {
        if (!sibling->reader_ || sibling->shape_.n_heads != n_heads || sibling->shape_.window != window || sibling->d_head_ != d_head_)
            throw std::runtime_error("reader: the sibling has other sizes");
        shared_plan_ = sibling->shared_plan_;
    }
}

Attention::Attention(const ca_head_shape& shape, int chunk_size, int memory_mb, bool share_prefix, int tpp_threshold,
                     torch::Dtype dtype, torch::Device device)
  : n_heads_(shape.n_heads), d_head_(shape.d_key), chunk_size_(chunk_size), memory_mb_(memory_mb),
    tpp_threshold_(tpp_threshold), shaped_(true), shape_(shape), share_prefix_(share_prefix),
    options_(torch::TensorOptions().dtype(dtype).layout(torch::kStrided).device(device).requires_grad(false)) {
    init();
}

void Attention::init() {
    if (!options_.device().is_cuda())
        throw std::runtime_error(
            "chunk_attn (B200 build) computes on CUDA devices only and has no CPU path: got device " +
            options_.device().str());
    if (n_heads_ <= 0 || d_head_ <= 0 || chunk_size_ <= 0 || memory_mb_ < 0)
        throw std::runtime_error("n_heads, d_head, chunk_size must be positive");
    const auto st = c10::typeMetaToScalarType(options_.dtype());
    if (st == torch::kFloat16) {
        ca_dtype_ = CA_DTYPE_F16;
    } else if (st == torch::kFloat32) {
        ca_dtype_ = CA_DTYPE_F32;
    } else if (st == torch::kBFloat16 && shaped_) {
        ca_dtype_ = CA_DTYPE_BF16;
    } else {
        throw std::runtime_error(std::string("unsupported dtype ") + c10::toString(st));
    }
    if (!options_.device().has_index())
        options_ = options_.device(torch::Device(torch::kCUDA, c10::cuda::current_device()));
    if (shaped_) {
        chunk_bytes_ = ca_chunk_bytes_shaped(&shape_, chunk_size_, ca_dtype_);
        if (chunk_bytes_ <= 0) throw std::runtime_error("n_kv_heads must divide n_heads, head sizes must lie in 1 .. 256");
        const int per16 = 16 / (ca_dtype_ == CA_DTYPE_F32 ? 4 : 2);
        k_padded_ = (shape_.d_key + per16 - 1) / per16 * per16;
        v_padded_ = (shape_.d_value + per16 - 1) / per16 * per16;
    } else {
        chunk_bytes_ = ca_chunk_bytes(n_heads_, d_head_, chunk_size_, ca_dtype_);
        k_padded_ = v_padded_ = d_head_;
    }
    // same sizing rule as the reference's allocator: as many whole chunks as memory_mb holds
    max_chunks_ = (int64_t)((double)memory_mb_ * 1024.0 * 1024.0 / (double)chunk_bytes_);
    c10::cuda::CUDAGuard guard(options_.device());
    if (!reader_) {
        pool_ = torch::empty({std::max<int64_t>(max_chunks_, 1) * chunk_bytes_}, options_.dtype(torch::kUInt8));
        tree_ = std::make_shared<PrefixTree>(chunk_size_, max_chunks_, chunk_bytes_, share_prefix_);
        tables_ = std::make_shared<Tables>();
    }
    check_rc(shaped_ ? ca_context_create_shaped(&ctx_, options_.device().index(), &shape_, chunk_size_, ca_dtype_,
                                                pool_.data_ptr(), max_chunks_, tpp_threshold_)
                     : ca_context_create(&ctx_, options_.device().index(), n_heads_, d_head_, chunk_size_, ca_dtype_,
                                         pool_.data_ptr(), max_chunks_, tpp_threshold_),
             "chunk_attn: context");
    valid_ = false;
    shared_plan_ = std::make_shared<SharedPlan>();
    shared_tables_ = std::make_shared<SharedTables>();
}

Attention::SharedPlan::~SharedPlan() {
    if (plan) ca_plan_destroy(plan);
}

Attention::~Attention() {
    if (worker_.joinable()) {
        {
            std::lock_guard<std::mutex> lock(worker_mutex_);
            worker_stop_ = true;
        }
        worker_cv_.notify_all();
        worker_.join();
    }
    if (ctx_) ca_context_destroy(ctx_);
}

void Attention::worker_loop() {
    for (;;) {
        std::function<void()> task;
        {
            std::unique_lock<std::mutex> lock(worker_mutex_);
            worker_cv_.wait(lock, [this] { return worker_stop_ || !worker_queue_.empty(); });
            if (worker_queue_.empty()) return;  // stop requested and nothing left to run
            task = std::move(worker_queue_.front());
            worker_queue_.pop_front();
        }
        task();
    }
}

void* Attention::stream() const {
    return c10::cuda::getCurrentCUDAStream(options_.device().index()).stream();
}

torch::Tensor Attention::to_cache(torch::Tensor t) const {
    if (t.device() != options_.device() || t.scalar_type() != c10::typeMetaToScalarType(options_.dtype()))
        t = t.to(options_);
    if (t.dim() > 0 && t.stride(t.dim() - 1) != 1) t = t.contiguous();
    return t;
}

void Attention::check_kv(const torch::Tensor& k, const torch::Tensor& v, int64_t n, const char* what) const {
    if (shape_.latent) throw std::runtime_error("a latent cache takes no separate keys and values");
    const int dv = shaped_ ? shape_.d_value : d_head_;
    if (k.dim() != 3 || v.dim() != 3 || k.size(0) != n || v.size(0) != n || k.size(1) != kv_heads() || v.size(1) != kv_heads() ||
        k.size(2) != d_head_ || v.size(2) != dv)
        throw std::runtime_error(what);
}

torch::Tensor Attention::pad_heads(torch::Tensor t, int padded) const {
    return t.size(2) == padded ? t : torch::constant_pad_nd(t, {0, padded - t.size(2)});
}

int Attention::add_seq(const std::vector<int>& tokens, torch::Tensor k, torch::Tensor v) {
    need_owner();
    check_kv(k, v, k.dim() > 0 ? k.size(0) : 0, "add_seq: k and v must be [n_tokens, n_heads, d_head]");
    // rows past the last token (a right-padded prompt) are ignored, as the reference's slices do
    if (k.size(0) < (int64_t)tokens.size()) throw std::runtime_error("add_seq: one K/V row per token is required");
    std::vector<NewChunk> created;
    const int seq_idx = tree_->add_seq(tokens, created);
    valid_ = false;
    if (!created.empty()) {
        // the new chunks hold one contiguous token range: a single scatter fills them all.  K/V of
        // the matched prefix are not read (the first sequence that brought a chunk wrote it).
        k = pad_heads(to_cache(k), k_padded_);
        v = pad_heads(to_cache(v), v_padded_);
        if (k.strides() != v.strides() || k_padded_ != v_padded_) {
            k = k.contiguous();
            v = v.contiguous();
        }
        std::vector<int32_t> ids;
        ids.reserve(created.size());
        int n_tokens = 0;
        for (const NewChunk& nc : created) {
            ids.push_back(nc.chunk->id);
            n_tokens += nc.n_tokens;
        }
        c10::cuda::CUDAGuard guard(options_.device());
        check_rc(ca_scatter_prefill(ctx_, k.data_ptr(), v.data_ptr(), k.stride(0), k.stride(1), created.front().token_start,
                                    n_tokens, ids.data(), stream()),
                 "add_seq");
    }
    return seq_idx;
}

std::shared_ptr<std::future<int>> Attention::add_seq_async(const std::vector<int>& tokens, torch::Tensor k,
                                                           torch::Tensor v) {
    // The reference declares this and throws (cpp/chunk_attn/attention.cpp:195-208).  Here the
    // insertion runs on this object's worker thread; the tensors are held by value until it is done.
    auto promise = std::make_shared<std::promise<int>>();
    auto future = std::make_shared<std::future<int>>(promise->get_future());
    const c10::cuda::CUDAStream caller_stream = c10::cuda::getCurrentCUDAStream(options_.device().index());
    {
        std::lock_guard<std::mutex> lock(worker_mutex_);
        if (!worker_.joinable()) worker_ = std::thread([this] { worker_loop(); });
        worker_queue_.emplace_back([this, promise, tokens, k, v, caller_stream]() mutable {
            try {
                c10::cuda::CUDAStreamGuard guard(caller_stream);  // the current stream is per thread
                promise->set_value(add_seq(tokens, k, v));
            } catch (...) {
                promise->set_exception(std::current_exception());
            }
            k.reset();
            v.reset();
        });
    }
    worker_cv_.notify_one();
    return future;
}

int Attention::append_completion(int seq_idx, const std::vector<int>& tokens, torch::Tensor k, torch::Tensor v) {
    need_owner();
    const int64_t n = (int64_t)tokens.size();
    check_kv(k, v, n, "append_completion: k and v must be [n_tokens, n_heads, d_head]");
    std::vector<std::pair<Chunk*, Chunk*>> pairs;
    std::vector<std::pair<Chunk*, int>> slots;
    tree_->append_completion(seq_idx, tokens, pairs, slots);
    valid_ = false;
    k = pad_heads(to_cache(k), k_padded_);
    v = pad_heads(to_cache(v), v_padded_);
    if (k.strides() != v.strides() || k_padded_ != v_padded_) {
        k = k.contiguous();
        v = v.contiguous();
    }
    c10::cuda::CUDAGuard guard(options_.device());
    if (!pairs.empty()) {  // copy-on-write of the forked leaf, before the beams diverge
        std::vector<int32_t> src, dst;
        for (auto& p : pairs) {
            src.push_back(p.first->id);
            dst.push_back(p.second->id);
        }
        check_rc(ca_copy_chunks(ctx_, src.data(), dst.data(), (int)src.size(), stream()), "append_completion");
    }
    std::vector<int32_t> ids, rows;
    for (auto& s : slots) {
        ids.push_back(s.first->id);
        rows.push_back(s.second);
    }
    check_rc(ca_scatter_rows(ctx_, k.data_ptr(), v.data_ptr(), k.stride(0), k.stride(1), (int)ids.size(), ids.data(),
                             rows.data(), stream()),
             "append_completion");
    return seq_idx;
}

void Attention::remove_seq(int seq_idx) {
    need_owner();
    tree_->remove_seq(seq_idx);
    valid_ = false;
}

std::vector<Chunk*> Attention::reserve() {
    need_owner();
    std::vector<Chunk*> fresh = tree_->reserve();
    if (!fresh.empty()) valid_ = false;
    return fresh;
}

namespace {
inline int64_t now_ns() {
    return std::chrono::duration_cast<std::chrono::nanoseconds>(std::chrono::steady_clock::now().time_since_epoch()).count();
}
}  // namespace

void Attention::refresh_kernel_context(bool force) {
    if (!force && valid_ && planned_version_ == tree_->version()) return;
    const int64_t t0 = now_ns();
    std::vector<ca_chunk_info> infos = tree_->get_chunks();
    const int64_t t1 = now_ns();
    c10::cuda::CUDAGuard guard(options_.device());
    SharedPlan& sp = *shared_plan_;
    const bool same = sp.plan != nullptr && sp.n_seqs == tree_->n_seqs() && sp.infos.size() == infos.size() &&
                      (infos.empty() || std::memcmp(sp.infos.data(), infos.data(), infos.size() * sizeof(ca_chunk_info)) == 0);
    if (!same) {
        sp.n_seqs = -1;  // nothing to reuse if the rebuild below is refused
        check_rc(ca_plan_build_for_context(ctx_, &sp.plan, infos.data(), (int)infos.size(), tree_->n_seqs()),
                 "refresh_kernel_context");
        sp.infos.swap(infos);
        sp.n_seqs = tree_->n_seqs();
        sp.builds++;
    } else {
        sp.reuses++;
    }
    const int64_t t2 = now_ns();
    check_rc(ca_refresh_from_plan(ctx_, sp.plan, stream()), "refresh_kernel_context");
    valid_ = true;
    planned_version_ = tree_->version();
    planned_appended_ = tree_->appended();
    const int64_t t3 = now_ns();
    host_times_.refreshes++;
    host_times_.walk_ns += t1 - t0;
    host_times_.plan_ns += t2 - t1;
    host_times_.upload_ns += t3 - t2;
}

std::vector<Chunk*> Attention::append_token(const std::vector<int>& tokens, torch::Tensor k, torch::Tensor v, bool) {
    if (tree_->tails().size() != tokens.size()) throw std::runtime_error("num of seqs is not equal to num of tokens");
    const int64_t n = (int64_t)tokens.size();
    check_kv(k, v, n, "append_token: k and v must be [n_seqs, n_heads, d_head]");
    std::vector<Chunk*> fresh = reserve();
    refresh_kernel_context(false);
    k = pad_heads(to_cache(k), k_padded_).contiguous();
    v = pad_heads(to_cache(v), v_padded_).contiguous();
    c10::cuda::CUDAGuard guard(options_.device());
    check_rc(ca_append_kv(ctx_, k.data_ptr(), v.data_ptr(), (int)n, stream()), "append_token");
    tree_->append_token_ids(tokens);
    return fresh;
}

void Attention::clear() {
    need_owner();
    tree_->clear();
    valid_ = false;
}

void Attention::duplicate(int seq_idx, int copies) {
    need_owner();
    std::vector<std::pair<Chunk*, Chunk*>> pairs;
    tree_->duplicate(seq_idx, copies, pairs);
    if (pairs.empty()) return;
    valid_ = false;
    std::vector<int32_t> src, dst;
    for (auto& p : pairs) {
        src.push_back(p.first->id);
        dst.push_back(p.second->id);
    }
    c10::cuda::CUDAGuard guard(options_.device());
    check_rc(ca_copy_chunks(ctx_, src.data(), dst.data(), (int)src.size(), stream()), "duplicate");
}

torch::Tensor Attention::forward(torch::Tensor q, int partition) {
    if (!q.is_contiguous()) throw std::runtime_error("q is not contiguous");
    if (q.dim() != 3 || q.size(1) != n_heads_ || q.size(2) != d_head_)
        throw std::runtime_error("forward: q must be [n_seqs, n_heads, d_head]");
    if (q.size(0) != (int64_t)tree_->n_seqs()) throw std::runtime_error("forward: one query row per live sequence is required");
    if (q.device() != options_.device() || q.scalar_type() != c10::typeMetaToScalarType(options_.dtype()))
        throw std::runtime_error("forward: q must have the dtype and device of the cache");
    if (partition < 0 || partition > 2) throw std::runtime_error("Unsupported partition type");
    c10::cuda::CUDAGuard guard(options_.device());
    torch::Tensor output = torch::empty({q.size(0), n_heads_, d_head_}, options_);
    refresh_kernel_context(false);
    check_rc(ca_attention(ctx_, q.data_ptr(), output.data_ptr(), (int)q.size(0), partition, stream()), "forward");
    return output;
}

torch::Tensor Attention::forward_host(torch::Tensor q, c10::optional<torch::Tensor> out, int partition) {
    const auto st = c10::typeMetaToScalarType(options_.dtype());
    if (q.is_cuda()) throw std::runtime_error("forward_host: q must be a CPU tensor (use forward for device tensors)");
    if (!q.is_contiguous()) throw std::runtime_error("q is not contiguous");
    if (q.dim() != 3 || q.size(1) != n_heads_ || q.size(2) != d_head_ || q.scalar_type() != st)
        throw std::runtime_error("forward_host: q must be [n_seqs, n_heads, d_head] with the dtype of the cache");
    if (q.size(0) != (int64_t)tree_->n_seqs()) throw std::runtime_error("forward: one query row per live sequence is required");
    if (partition < 0 || partition > 2) throw std::runtime_error("Unsupported partition type");
    torch::Tensor result;
    if (out.has_value()) {
        result = *out;
        if (result.is_cuda() || !result.is_contiguous() || result.sizes() != q.sizes() || result.scalar_type() != st)
            throw std::runtime_error("forward_host: out must be a contiguous CPU tensor shaped and typed like q");
    } else {
        result = torch::empty(q.sizes(), torch::TensorOptions().dtype(st).device(torch::kCPU).pinned_memory(true));
    }
    c10::cuda::CUDAGuard guard(options_.device());
    refresh_kernel_context(false);
    check_rc(ca_attention_host(ctx_, q.data_ptr(), result.data_ptr(), (int)q.size(0), partition, stream()), "forward_host");
    return result;
}

void Attention::forward_to_peers(torch::Tensor q, const std::vector<int64_t>& peer_out_ptrs, int total_heads,
                                 int head_offset, int64_t multicast_ptr) {
    if (!q.is_contiguous()) throw std::runtime_error("q is not contiguous");
    if (q.dim() != 3 || q.size(0) != (int64_t)tree_->n_seqs() || q.size(1) != n_heads_ || q.size(2) != d_head_ ||
        q.device() != options_.device() || q.scalar_type() != c10::typeMetaToScalarType(options_.dtype()))
        throw std::runtime_error("forward_to_peers: q must be [n_seqs, n_heads, d_head] with the dtype and device of the cache");
    std::vector<void*> ptrs;
    for (int64_t p : peer_out_ptrs) ptrs.push_back(reinterpret_cast<void*>(p));
    c10::cuda::CUDAGuard guard(options_.device());
    refresh_kernel_context(false);
    check_rc(ca_attention_to_peers(ctx_, q.data_ptr(), ptrs.data(), (int)ptrs.size(), reinterpret_cast<void*>(multicast_ptr),
                                   total_heads, head_offset, (int)q.size(0), stream()),
             "forward_to_peers");
}

std::vector<int> Attention::extend(const std::vector<int>& rows, const std::vector<std::vector<int>>& tokens) {
    need_owner();
    const size_t n = rows.size();
    if (tokens.size() != n) throw std::runtime_error("extend: one token list per row is required");
    // everything that can be refused is refused before anything changes
    std::vector<char> seen(tree_->n_seqs(), 0);
    int64_t need = 0;
    for (size_t i = 0; i < n; i++) {
        if (tokens[i].empty()) throw std::runtime_error("extend: an entry has no tokens");
        if (rows[i] >= 0) {
            need += tree_->extend_need(rows[i], (int)tokens[i].size());
            if (seen[rows[i]]++) throw std::runtime_error("extend: a row is named twice");
        } else {
            need += (int64_t)tokens[i].size() / chunk_size_ + 1;
        }
    }
    if (tree_->pool().max_chunks() - tree_->pool().in_use() < need) throw std::runtime_error("ChunkAllocator: capacity reached");
    valid_ = false;
    tables_->n_tokens = -1;

    std::vector<int> out(rows);
    std::vector<std::vector<int32_t>> slot_of(n);
    std::vector<Chunk*> tail(n);
    for (size_t i = 0; i < n; i++) {
        if (rows[i] < 0) continue;
        std::vector<std::pair<Chunk*, int>> slots;
        tree_->extend_seq(rows[i], tokens[i], slots);
        for (const auto& s : slots) slot_of[i].push_back(s.first->id * chunk_size_ + s.second);
        tail[i] = tree_->tails()[rows[i]];
    }
    for (size_t i = 0; i < n; i++) {
        if (rows[i] >= 0) continue;
        std::vector<NewChunk> created;
        out[i] = tree_->add_seq(tokens[i], created);
        slot_of[i].assign(tokens[i].size(), -1);  // tokens of a matched prefix are in the pool already
        for (const NewChunk& nc : created)
            for (int j = 0; j < nc.n_tokens; j++) slot_of[i][nc.token_start + j] = nc.chunk->id * chunk_size_ + j;
        tail[i] = tree_->tails()[out[i]];
    }

    // tables: tok_slot | path_off | path_chunks | blocks (16-byte aligned)
    std::vector<int32_t> data;
    for (const auto& s : slot_of) data.insert(data.end(), s.begin(), s.end());
    tables_->path_off = (int64_t)data.size();
    std::vector<int32_t> off{0}, chunks;
    tables_->starts.assign(n, 0);
    tables_->lens.assign(n, 0);
    for (size_t i = 0; i < n; i++) {
        const size_t b = chunks.size();
        tables_->lens[i] = (int)tokens[i].size();
        tables_->starts[i] = -tables_->lens[i];
        for (Chunk* c = tail[i]; c->parent != nullptr; c = c->parent) {
            chunks.push_back(c->id);
            tables_->starts[i] += c->n_tokens();
        }
        std::reverse(chunks.begin() + b, chunks.end());
        off.push_back((int32_t)chunks.size());
    }
    data.insert(data.end(), off.begin(), off.end());
    tables_->path_chunks = (int64_t)data.size();
    data.insert(data.end(), chunks.begin(), chunks.end());
    while (data.size() % 4) data.push_back(0);
    tables_->blocks = (int64_t)data.size();
    tables_->block_rows = shape_.latent ? ca_latent_block(&shape_) : ca_rows_block(&shape_);
    tables_->n_blocks = 0;
    int32_t base = 0;
    for (size_t i = 0; i < n; i++) {
        const int len = (int)tokens[i].size();
        // the last blocks of a portion see the most context: they go first
        for (int b = (len - 1) / tables_->block_rows; b >= 0; b--) {
            const int lo = b * tables_->block_rows, hi = std::min(len, lo + tables_->block_rows);
            data.insert(data.end(), {(int32_t)i, base + lo, base + hi, 0});
            tables_->n_blocks++;
        }
        base += len;
    }
    data.insert(data.end(), tables_->starts.begin(), tables_->starts.end());
    c10::cuda::CUDAGuard guard(options_.device());
    SharedTables& st = *shared_tables_;
    if (!st.device.defined() || st.data != data) {
        torch::Tensor host = torch::empty({(int64_t)data.size()}, torch::TensorOptions().dtype(torch::kInt32).pinned_memory(true));
        std::memcpy(host.data_ptr(), data.data(), data.size() * sizeof(int32_t));
        st.device = host.to(options_.device(), torch::kInt32, /*non_blocking=*/true);
        st.data.swap(data);
        st.blocks.clear();
        st.windows.clear();
    }
    tables_->device = st.device;
    tables_->n_tokens = base;
    return out;
}

namespace {
const float* f32_ptr(const c10::optional<torch::Tensor>& t, int64_t n, const char* msg) {
    if (!t.has_value()) return nullptr;
    if (!t->is_cuda() || t->scalar_type() != torch::kFloat32 || !t->is_contiguous() || t->numel() != n) throw std::runtime_error(msg);
    return t->data_ptr<float>();
}
const int32_t* i32_ptr(const torch::Tensor& t, int64_t n, const char* msg) {
    if (!t.is_cuda() || t.scalar_type() != torch::kInt32 || !t.is_contiguous() || t.numel() != n) throw std::runtime_error(msg);
    return t.data_ptr<int32_t>();
}
}  // namespace

torch::Tensor Attention::store_qkv(torch::Tensor qkv, torch::Tensor positions, c10::optional<torch::Tensor> q_norm,
                                   c10::optional<torch::Tensor> k_norm, double eps, int rot_dims,
                                   c10::optional<torch::Tensor> key_freq, c10::optional<torch::Tensor> value_freq,
                                   c10::optional<std::vector<int>> append_tokens) {
    if (!shaped_) throw std::runtime_error("store_qkv needs a cache with a head shape");
    const int64_t n = qkv.dim() == 2 ? qkv.size(0) : -1;
    if (n < 0 || qkv.size(1) < (int64_t)(n_heads_ + kv_heads()) * d_head_ + (int64_t)kv_heads() * shape_.d_value || qkv.stride(1) != 1 ||
        qkv.device() != options_.device() || qkv.scalar_type() != c10::typeMetaToScalarType(options_.dtype()))
        throw std::runtime_error("store_qkv: qkv must be [n_tokens, q | k | v heads] with the dtype and device of the cache");
    ca_qkv_args a{};
    a.qkv = qkv.data_ptr();
    a.row_stride = qkv.stride(0);
    a.q_norm = f32_ptr(q_norm, d_head_, "store_qkv: q_norm must be fp32 [d_key]");
    a.k_norm = f32_ptr(k_norm, d_head_, "store_qkv: k_norm must be fp32 [d_key]");
    a.eps = (float)eps;
    a.rot_dims = rot_dims;
    a.key_freq = f32_ptr(key_freq, rot_dims / 2, "store_qkv: key_freq must be fp32 [rot_dims / 2]");
    a.value_freq = f32_ptr(value_freq, shape_.d_value / 2, "store_qkv: value_freq must be fp32 [d_value / 2]");
    a.positions = i32_ptr(positions, n, "store_qkv: positions must be int32 [n_tokens]");
    a.n_tokens = (int32_t)n;
    c10::cuda::CUDAGuard guard(options_.device());
    torch::Tensor q = torch::empty({n, n_heads_, k_padded_}, options_);
    a.q_out = q.data_ptr();
    if (append_tokens.has_value()) {
        if (tree_->tails().size() != append_tokens->size() || (int64_t)append_tokens->size() != n)
            throw std::runtime_error("num of seqs is not equal to num of tokens");
        reserve();
        refresh_kernel_context(false);
        check_rc(ca_store_qkv(ctx_, &a, stream()), "store_qkv");
        tree_->append_token_ids(*append_tokens);
    } else {
        if (tables_->n_tokens != n) throw std::runtime_error("store_qkv: extend must have described these tokens");
        a.tok_slot = tables_->device.data_ptr<int32_t>();
        check_rc(ca_store_qkv(ctx_, &a, stream()), "store_qkv");
    }
    return q;
}

torch::Tensor Attention::forward_rows(torch::Tensor q, torch::Tensor positions, c10::optional<torch::Tensor> value_freq,
                                      c10::optional<torch::Tensor> row_entry) {
    if (!shaped_) throw std::runtime_error("forward_rows needs a cache with a head shape");
    if (q.dim() != 3 || q.size(1) != n_heads_ || q.size(2) != k_padded_ || !q.is_contiguous() || q.device() != options_.device() ||
        q.scalar_type() != c10::typeMetaToScalarType(options_.dtype()))
        throw std::runtime_error("forward_rows: q must be what store_qkv returned");
    const int64_t n = q.size(0);
    c10::cuda::CUDAGuard guard(options_.device());
    torch::Tensor out = torch::empty({n, n_heads_, shape_.d_value}, options_);
    ca_rows_args a{};
    a.q = q.data_ptr();
    a.out = out.data_ptr();
    a.n_rows = (int32_t)n;
    a.positions = i32_ptr(positions, n, "forward_rows: positions must be int32 [n_rows]");
    a.value_freq = f32_ptr(value_freq, shape_.d_value / 2, "forward_rows: value_freq must be fp32 [d_value / 2]");
    if (row_entry.has_value()) {
        if (tables_->n_tokens != n) throw std::runtime_error("forward_rows: extend must have described these tokens");
        const int32_t* t = tables_->device.data_ptr<int32_t>();
        a.row_entry = i32_ptr(*row_entry, n, "forward_rows: row_entry must be int32 [n_rows]");
        a.path_off = t + tables_->path_off;
        a.path_chunks = t + tables_->path_chunks;
        a.blocks = t + tables_->blocks;
        a.n_blocks = tables_->n_blocks;
        a.block_rows = tables_->block_rows;
    } else {
        refresh_kernel_context(false);
    }
    check_rc(ca_attention_rows(ctx_, &a, stream()), "forward_rows");
    return out;
}

// ---- latent caches ------------------------------------------------------------------------------------------------------

void Attention::need_latent(const char* what) const {
    if (!shape_.latent) throw std::runtime_error(std::string(what) + " needs a latent cache");
}
void Attention::need_owner() const {
    if (reader_) throw std::runtime_error("a reader does not change the cache it reads");
}

namespace {
torch::Tensor upload(const std::vector<int32_t>& data, torch::Device device) {
    torch::Tensor host = torch::empty({(int64_t)data.size()}, torch::TensorOptions().dtype(torch::kInt32).pinned_memory(true));
    std::memcpy(host.data_ptr(), data.data(), data.size() * sizeof(int32_t));
    return host.to(device, torch::kInt32, /*non_blocking=*/true);
}
}  // namespace

// {entry, first row, end row, 0} of runs of at most block_rows rows
const std::pair<torch::Tensor, int>& Attention::blocks_of(int block_rows) {
    auto& all = shared_tables_->blocks;
    auto f = all.find(block_rows);
    if (f != all.end()) return f->second;
    std::vector<int32_t> data;
    int32_t base = 0;
    for (size_t i = 0; i < tables_->lens.size(); i++) {
        const int len = tables_->lens[i];
        for (int b = 0; b < len; b += block_rows) data.insert(data.end(), {(int32_t)i, base + b, base + std::min(len, b + block_rows), 0});
        base += len;
    }
    return all.emplace(block_rows, std::make_pair(upload(data, options_.device()), (int)(data.size() / 4))).first->second;
}

const Attention::WindowTables& Attention::window_tables() {
    auto& all = shared_tables_->windows;
    auto f = all.find(shape_.window);
    if (f != all.end()) return f->second;
    const size_t E = tables_->lens.size();
    WindowTables w;
    std::vector<int32_t> src, base{0}, first;
    for (size_t i = 0; i < E; i++) {
        const int64_t start = tables_->starts[i], len = tables_->lens[i], win = shape_.window > 0 ? shape_.window : start + len;
        first.push_back((int32_t)std::max<int64_t>(0, start - win + 1));
        base.push_back(base.back() + (int32_t)(start + len - first.back()));
        // positions start .. start + len - 1 see min(position + 1, win) tokens each
        const int64_t growing = std::min(len, std::max<int64_t>(0, win - start));
        w.pairs += growing * (2 * start + growing + 1) / 2 + (len - growing) * win;
        const int32_t* path = shared_tables_->data.data() + tables_->path_chunks + shared_tables_->data[tables_->path_off + (int64_t)i];
        for (int64_t pos = first.back(); pos < start + len; pos++) src.push_back(path[pos / chunk_size_] * chunk_size_ + (int32_t)(pos % chunk_size_));
    }
    w.rows = base.back();
    src.insert(src.end(), base.begin(), base.end());
    src.insert(src.end(), first.begin(), first.end());
    w.device = upload(src, options_.device());
    return all.emplace(shape_.window, w).first->second;
}

std::pair<int64_t, int64_t> Attention::window_load() {
    need_latent("window_load");
    if (tables_->n_tokens < 0) throw std::runtime_error("window_load: extend must have described the tokens");
    const WindowTables& w = window_tables();
    return {w.rows, w.pairs};
}

torch::Tensor Attention::store_latent(torch::Tensor in, torch::Tensor positions, torch::Tensor q_norm, torch::Tensor kv_norm, double eps,
                                      c10::optional<torch::Tensor> freq, c10::optional<std::vector<int>> append_tokens) {
    need_latent("store_latent");
    need_owner();
    const int64_t q_rank = q_norm.numel(), rot = shape_.d_key - shape_.d_value;
    const int64_t n = in.dim() == 2 ? in.size(0) : -1;
    if (n < 1 || in.size(1) < q_rank + shape_.d_key || in.stride(1) != 1 || in.device() != options_.device() ||
        in.scalar_type() != c10::typeMetaToScalarType(options_.dtype()))
        throw std::runtime_error("store_latent: [n_tokens, query latent | latent | shared key part] with the dtype and device of the cache is required");
    ca_latent_store_args a{};
    a.in = in.data_ptr();
    a.row_stride = in.stride(0);
    a.q_rank = (int32_t)q_rank;
    a.q_norm = f32_ptr(q_norm, q_rank, "store_latent: q_norm must be fp32 [q_rank]");
    a.kv_norm = f32_ptr(kv_norm, shape_.d_value, "store_latent: kv_norm must be fp32 [latent size]");
    a.eps = (float)eps;
    a.freq = f32_ptr(freq, rot, "store_latent: freq must be fp32 [2, rotated / 2]");
    a.positions = i32_ptr(positions, n, "store_latent: positions must be int32 [n_tokens]");
    a.n_tokens = (int32_t)n;
    c10::cuda::CUDAGuard guard(options_.device());
    torch::Tensor q = torch::empty({n, q_rank}, options_);
    a.q_out = q.data_ptr();
    if (append_tokens.has_value()) {
        if (tree_->tails().size() != append_tokens->size() || (int64_t)append_tokens->size() != n)
            throw std::runtime_error("num of seqs is not equal to num of tokens");
        reserve();
        refresh_kernel_context(false);
        check_rc(ca_latent_store(ctx_, &a, stream()), "store_latent");
        tree_->append_token_ids(*append_tokens);
    } else {
        if (tables_->n_tokens != n) throw std::runtime_error("store_latent: extend must have described these tokens");
        a.tok_slot = tables_->device.data_ptr<int32_t>();
        check_rc(ca_latent_store(ctx_, &a, stream()), "store_latent");
    }
    return q;
}

torch::Tensor Attention::forward_latent(torch::Tensor q_lat, torch::Tensor q, torch::Tensor positions, c10::optional<torch::Tensor> freq,
                                        c10::optional<torch::Tensor> sink, c10::optional<torch::Tensor> row_entry) {
    need_latent("forward_latent");
    const int64_t rot = shape_.d_key - shape_.d_value;
    const auto st = c10::typeMetaToScalarType(options_.dtype());
    if (q_lat.dim() != 3 || q_lat.size(1) != n_heads_ || q_lat.size(2) != shape_.d_value || !q_lat.is_contiguous() ||
        q_lat.device() != options_.device() || q_lat.scalar_type() != st)
        throw std::runtime_error("forward_latent: q_lat must be contiguous [n_rows, n_heads, latent size] with the dtype and device of the cache");
    const int64_t n = q_lat.size(0);
    if (q.dim() != 3 || q.size(0) != n || q.size(1) != n_heads_ || q.size(2) < rot || q.stride(2) != 1 || q.device() != options_.device() ||
        q.scalar_type() != st)
        throw std::runtime_error("forward_latent: q must be [n_rows, n_heads, unrotated + rotated] like q_lat");
    c10::cuda::CUDAGuard guard(options_.device());
    torch::Tensor out = torch::empty_like(q_lat);
    ca_latent_args a{};
    a.q_lat = q_lat.data_ptr();
    a.q_rot = static_cast<const char*>(q.data_ptr()) + (q.size(2) - rot) * q.element_size();
    a.q_rot_row = q.stride(0);
    a.q_rot_head = q.stride(1);
    a.out = out.data_ptr();
    a.n_rows = (int32_t)n;
    a.positions = i32_ptr(positions, n, "forward_latent: positions must be int32 [n_rows]");
    a.freq = f32_ptr(freq, rot, "forward_latent: freq must be fp32 [2, rotated / 2]");
    a.sink = f32_ptr(sink, n_heads_, "forward_latent: sink must be fp32 [n_heads]");
    a.delta_tokens = -1;
    if (row_entry.has_value()) {
        if (tables_->n_tokens != n) throw std::runtime_error("forward_latent: extend must have described these tokens");
        const int32_t* t = tables_->device.data_ptr<int32_t>();
        a.block_rows = ca_latent_block(&shape_);
        const auto& blocks = blocks_of(a.block_rows);
        a.row_entry = i32_ptr(*row_entry, n, "forward_latent: row_entry must be int32 [n_rows]");
        a.path_off = t + tables_->path_off;
        a.path_chunks = t + tables_->path_chunks;
        a.blocks = blocks.first.data_ptr<int32_t>();
        a.n_blocks = blocks.second;
    } else {
        refresh_kernel_context(false);
        a.delta_tokens = (int32_t)(tree_->appended() - planned_appended_);
    }
    check_rc(ca_latent_attention(ctx_, &a, stream()), "forward_latent");
    return out;
}

std::pair<torch::Tensor, torch::Tensor> Attention::gather_latents() {
    need_latent("gather_latents");
    if (tables_->n_tokens < 0) throw std::runtime_error("gather_latents: extend must have described the tokens");
    c10::cuda::CUDAGuard guard(options_.device());
    const WindowTables& w = window_tables();
    const int64_t pad = (shape_.d_key - shape_.d_value + 63) / 64 * 64;
    torch::Tensor lat = torch::empty({w.rows, shape_.d_value}, options_), rot = torch::empty({w.rows, std::max<int64_t>(pad, 64)}, options_);
    const int32_t* t = w.device.data_ptr<int32_t>();
    ca_latent_gather_args a{};
    a.lat = lat.data_ptr();
    a.rot = rot.data_ptr();
    a.rot_stride = (int32_t)rot.size(1);
    a.n_rows = (int32_t)w.rows;
    a.src_row = t;
    check_rc(ca_latent_gather(ctx_, &a, stream()), "gather_latents");
    return {lat, rot};
}

torch::Tensor Attention::forward_expanded(torch::Tensor q, torch::Tensor kv, torch::Tensor rot, torch::Tensor positions,
                                          c10::optional<torch::Tensor> freq, c10::optional<torch::Tensor> sink, int vdim) {
    need_latent("forward_expanded");
    const int64_t rotated = shape_.d_key - shape_.d_value, n = q.size(0);
    const auto st = c10::typeMetaToScalarType(options_.dtype());
    if (q.dim() != 3 || q.size(1) != n_heads_ || q.size(2) <= rotated || !q.is_contiguous() || q.device() != options_.device() || q.scalar_type() != st)
        throw std::runtime_error("forward_expanded: q must be contiguous [n_rows, n_heads, unrotated + rotated] with the dtype and device of the cache");
    if (tables_->n_tokens != n) throw std::runtime_error("forward_expanded: extend must have described these tokens");
    const int dim = (int)(q.size(2) - rotated);
    c10::cuda::CUDAGuard guard(options_.device());
    const WindowTables& w = window_tables();
    if (kv.dim() != 2 || kv.size(0) != w.rows || kv.size(1) != (int64_t)n_heads_ * (dim + vdim) || kv.stride(1) != 1 || kv.device() != options_.device() ||
        kv.scalar_type() != st || rot.dim() != 2 || rot.size(0) != w.rows || !rot.is_contiguous() || rot.device() != options_.device() || rot.scalar_type() != st)
        throw std::runtime_error("forward_expanded: kv must be [window rows, n_heads * (dim + vdim)], rot what gather_latents returned");
    torch::Tensor out = torch::empty({n, n_heads_, vdim}, options_);
    const auto& blocks = blocks_of(ca_latent_expanded_block());
    const int32_t* t = w.device.data_ptr<int32_t>();
    ca_latent_expanded_args a{};
    a.q = q.data_ptr();
    a.kv = kv.data_ptr();
    a.kv_rows = w.rows;
    a.kv_stride = kv.stride(0);
    a.rot = rot.data_ptr();
    a.rot_stride = (int32_t)rot.size(1);
    a.out = out.data_ptr();
    a.n_rows = (int32_t)n;
    a.dim = dim;
    a.vdim = vdim;
    a.positions = i32_ptr(positions, n, "forward_expanded: positions must be int32 [n_rows]");
    a.freq = f32_ptr(freq, rotated, "forward_expanded: freq must be fp32 [2, rotated / 2]");
    a.sink = f32_ptr(sink, n_heads_, "forward_expanded: sink must be fp32 [n_heads]");
    a.base = t + w.rows;
    a.first = t + w.rows + (int64_t)tables_->lens.size() + 1;
    a.blocks = blocks.first.data_ptr<int32_t>();
    a.n_blocks = blocks.second;
    check_rc(ca_latent_expanded(ctx_, &a, stream()), "forward_expanded");
    return out;
}

void Attention::print(Chunk* root, int level) {
    if (root == nullptr) root = tree_->root();
    std::string indent(4 * level, ' ');
    std::cout << indent << root->to_string(true) << std::endl;
    for (Chunk* child : root->children) print(child, level + 1);
}

ca_plan_stats Attention::plan_stats() {
    refresh_kernel_context(false);
    ca_plan_stats st;
    check_rc(ca_context_stats(ctx_, &st), "plan_stats");
    return st;
}

void Attention::set_option(int option, int64_t value) {
    check_rc(ca_context_set_option(ctx_, option, value), "set_option");
    valid_ = false;
    shared_plan_ = std::make_shared<SharedPlan>();  // its work lists now differ from its siblings'
}

void Attention::attn_partials(torch::Tensor q, int phases) {
    if (!q.is_contiguous() || q.dim() != 3 || q.size(0) != (int64_t)tree_->n_seqs() || q.size(1) != n_heads_ ||
        q.size(2) != d_head_ || q.device() != options_.device() ||
        q.scalar_type() != c10::typeMetaToScalarType(options_.dtype()))
        throw std::runtime_error("attn_partials: q must be a contiguous [n_seqs, n_heads, d_head] tensor of the cache's dtype and device");
    c10::cuda::CUDAGuard guard(options_.device());
    refresh_kernel_context(false);
    check_rc(ca_attn_partials(ctx_, q.data_ptr(), (int)q.size(0), phases, stream()), "attn_partials");
}

void Attention::attn_merge(torch::Tensor out) {
    if (!out.is_contiguous() || out.dim() != 3 || out.size(0) != (int64_t)tree_->n_seqs() || out.size(1) != n_heads_ ||
        out.size(2) != d_head_ || out.device() != options_.device() ||
        out.scalar_type() != c10::typeMetaToScalarType(options_.dtype()))
        throw std::runtime_error("attn_merge: out must be a contiguous [n_seqs, n_heads, d_head] tensor of the cache's dtype and device");
    c10::cuda::CUDAGuard guard(options_.device());
    check_rc(ca_attn_merge(ctx_, out.data_ptr(), (int)out.size(0), stream()), "attn_merge");
}

int Attention::device_status() {
    int32_t st = 0;
    c10::cuda::CUDAGuard guard(options_.device());
    const int rc = ca_status_read(ctx_, stream(), &st);
    if (rc != CA_OK && rc != CA_ERR_DEVICE_STATUS) check_rc(rc, "device_status");
    return st;
}

}  // namespace ca_host

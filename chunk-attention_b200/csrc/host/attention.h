// ca_host::Attention — the C++ object behind chunk_attn.Attention.
//
// Same constructor arguments, methods, row-order contract and error messages as the reference's
// GPT::Attention (cpp/chunk_attn/attention.h:16-75, cpp/chunk_attn/attention.cpp), so that the
// reference's llama_hf model and ModelHost drive it unchanged.  Differences in substance:
// K/V live in ONE device allocation in the library's private tile layout and every data-path
// operation (prefill scatter, token append, copy-on-write, attention) is a CUDA kernel behind
// the C ABI of include/chunk_attn_b200.h, launched on torch's current stream.  There is no CPU
// implementation: constructing it on a non-CUDA device throws.
#pragma once
#include <torch/torch.h>

#include <condition_variable>
#include <deque>
#include <functional>
#include <future>
#include <map>
#include <memory>
#include <mutex>
#include <thread>
#include <vector>

#include "../../../include/chunk_attn_b200.h"
#include "prefix_tree.h"

namespace ca_host {

class Attention {
  public:
    Attention(int n_heads, int d_head, int chunk_size, int memory_mb = 2048, bool share_prefix = true,
              int tpp_threshold = 1, torch::Dtype dtype = torch::kFloat16,
              torch::Device device = torch::Device(torch::kCUDA));
    // heads described by a ca_head_shape (grouped key/value heads, values of another width, a unit term in the
    // softmax denominator, any scale): the cache of layers driven through extend / store_qkv / forward_rows
    Attention(const ca_head_shape& shape, int chunk_size, int memory_mb, bool share_prefix, int tpp_threshold,
              torch::Dtype dtype, torch::Device device);
    // same configuration, fresh empty cache (one per transformer layer in the reference's model)
    Attention(Attention& other);
    // A second view of a latent cache for a layer that reads what `source` stores, with query heads, a scale and a window of
    // its own: pool, tree and the tables of the current portions are the source's, and only the source changes them.
    // `sibling`: a reader of the same sizes whose work lists are shared.
    Attention(Attention& source, int n_heads, double scale, int window, Attention* sibling);
    ~Attention();
    Attention& operator=(const Attention&) = delete;

    int add_seq(const std::vector<int>& tokens, torch::Tensor k, torch::Tensor v);
    // add_seq on a worker thread of this object; the kernels go to the stream that is current on the
    // calling thread now.  Insertions run in the order they were queued.  Until the future is ready
    // no other method of this object may be called (the tree is not locked).
    std::shared_ptr<std::future<int>> add_seq_async(const std::vector<int>& tokens, torch::Tensor k, torch::Tensor v);
    void remove_seq(int seq_idx);
    // One step of portions, tree side: entry i brings the next tokens of row rows[i] as the rows are now, or of a new
    // sequence (rows[i] < 0).  Returns the row of each entry (a new one's at the moment it was inserted, existing ones
    // are handled first).  store_qkv and forward_rows then work on these entries' tokens, laid end to end, until the
    // next change of the tree.
    std::vector<int> extend(const std::vector<int>& rows, const std::vector<std::vector<int>>& tokens);
    // Projections [n_tokens, q heads | k heads | v heads] to attention operands: k and v go into the pool, q is returned
    // ([n_tokens, n_heads, padded d_key]).  With append_tokens: one token per row, appended to every row as
    // append_token does.
    torch::Tensor store_qkv(torch::Tensor qkv, torch::Tensor positions, c10::optional<torch::Tensor> q_norm,
                            c10::optional<torch::Tensor> k_norm, double eps, int rot_dims, c10::optional<torch::Tensor> key_freq,
                            c10::optional<torch::Tensor> value_freq, c10::optional<std::vector<int>> append_tokens);
    // [n_rows, n_heads, d_value]: decode over every row (row_entry not given), or the tokens of the last extend
    torch::Tensor forward_rows(torch::Tensor q, torch::Tensor positions, c10::optional<torch::Tensor> value_freq,
                               c10::optional<torch::Tensor> row_entry);
    // ---- latent caches ----
    // Projections [n_tokens, query latent | key/value latent | shared key part] to the pool; returns the normalised query
    // latents [n_tokens, q_rank].  append_tokens as in store_qkv.
    torch::Tensor store_latent(torch::Tensor in, torch::Tensor positions, torch::Tensor q_norm, torch::Tensor kv_norm, double eps,
                               c10::optional<torch::Tensor> freq, c10::optional<std::vector<int>> append_tokens);
    // q_lat [n_rows, n_heads, latent size]: queries in the latent space; q [n_rows, n_heads, unrotated + rotated], whose last
    // part is used.  Returns [n_rows, n_heads, latent size].  row_entry as in forward_rows.
    torch::Tensor forward_latent(torch::Tensor q_lat, torch::Tensor q, torch::Tensor positions, c10::optional<torch::Tensor> freq,
                                 c10::optional<torch::Tensor> sink, c10::optional<torch::Tensor> row_entry);
    // whether decode steps may leave row_entry out (bf16, 64-token chunks); otherwise every step is given by extend
    bool latent_decodes() const { return ca_latent_decodes(ctx_) != 0; }
    // What the current portions read: (rows of their windows in the cache, (query, key) pairs inside the windows)
    std::pair<int64_t, int64_t> window_load();
    // Those rows, laid out densely: latents [rows, latent size] and shared key parts [rows, padded to 64]
    std::pair<torch::Tensor, torch::Tensor> gather_latents();
    // whether forward_expanded serves heads of these sizes
    bool latent_expands(int dim, int vdim) const { return ca_latent_expands(ctx_, dim, vdim) != 0; }
    // Attention of the current portions over keys and values expanded from the gathered rows: kv [rows, n_heads * (dim +
    // vdim)], keys of all heads, then values; rot as gather_latents returns it.  Returns [n_rows, n_heads, vdim].
    torch::Tensor forward_expanded(torch::Tensor q, torch::Tensor kv, torch::Tensor rot, torch::Tensor positions,
                                   c10::optional<torch::Tensor> freq, c10::optional<torch::Tensor> sink, int vdim);
    std::vector<Chunk*> append_token(const std::vector<int>& tokens, torch::Tensor k, torch::Tensor v, bool fused = true);
    void refresh_kernel_context(bool force = false);
    std::vector<Chunk*> reserve();
    void clear();
    int64_t peak_memory_allocated() const { return tree_->pool().peak_memory_allocated(); }
    void duplicate(int seq_idx, int copies);
    // One beam-search step for row seq_idx: it forks into tokens.size() rows (seq_idx, seq_idx + 1, ...),
    // row seq_idx + i continuing with tokens[i] whose K/V are k[i], v[i] ([n_tokens, n_heads, d_head]).
    // Returns seq_idx.
    int append_completion(int seq_idx, const std::vector<int>& tokens, torch::Tensor k, torch::Tensor v);
    torch::Tensor forward(torch::Tensor q, int partition = 0);
    // forward for queries in host memory: returns a CPU tensor (written into `out` when given).  Pinned
    // tensors are used in place, the result rows are stored into host memory by the last kernel, and
    // the call returns when they are there.
    torch::Tensor forward_host(torch::Tensor q, c10::optional<torch::Tensor> out, int partition = 0);
    // head-sharded forward: rows are written into every rank's full-width output buffer (device
    // addresses this GPU can reach), this cache's heads landing at head_offset of total_heads
    // multicast_ptr != 0: a multicast address mapping the same buffer on every rank; rows are then written with one
    // multimem.st each instead of one store per rank
    void forward_to_peers(torch::Tensor q, const std::vector<int64_t>& peer_out_ptrs, int total_heads, int head_offset,
                          int64_t multicast_ptr = 0);

    Chunk* get_trie() { return tree_->root(); }
    std::vector<Chunk*> tails() { return tree_->tails(); }
    void print(Chunk* root = nullptr, int level = 0);
    std::vector<ca_chunk_info> get_chunks() { return tree_->get_chunks(); }

    // introspection used by the benchmark and the tests
    ca_plan_stats plan_stats();
    void set_option(int option, int64_t value);
    int device_status();
    // (plans built, plans reused) by this cache and the caches it shares its work lists with
    std::pair<int64_t, int64_t> plan_sharing() const { return {shared_plan_->builds, shared_plan_->reuses}; }
    // host time spent bringing the work lists up to date since the object was made: the tree walk (get_chunks),
    // planning (or finding the shared plan current) and the upload, in nanoseconds, and how many refreshes
    struct HostTimes { int64_t refreshes = 0, walk_ns = 0, plan_ns = 0, upload_ns = 0; };
    HostTimes host_times() const { return host_times_; }
    // the two launches of forward(), separately (per-kernel timing)
    void attn_partials(torch::Tensor q, int phases);
    void attn_merge(torch::Tensor out);

  private:
    void init();
    void* stream() const;
    torch::Tensor to_cache(torch::Tensor t) const;  // dtype/device of the cache, last dim contiguous

    int kv_heads() const { return shaped_ ? shape_.n_kv_heads : n_heads_; }
    torch::Tensor pad_heads(torch::Tensor t, int padded) const;  // zeros up to the pool's head size
    void check_kv(const torch::Tensor& k, const torch::Tensor& v, int64_t n, const char* what) const;

    int n_heads_, d_head_, chunk_size_, memory_mb_, tpp_threshold_;
    bool shaped_ = false;
    ca_head_shape shape_{};
    int k_padded_ = 0, v_padded_ = 0;  // head sizes in the pool
    bool share_prefix_;
    torch::TensorOptions options_;
    int ca_dtype_ = 0;
    int64_t max_chunks_ = 0;
    int64_t chunk_bytes_ = 0;
    torch::Tensor pool_;  // one uint8 tensor: [max_chunks][n_heads][K|V][chunk_size][d_head]
    std::shared_ptr<PrefixTree> tree_;
    bool reader_ = false;  // pool and tree belong to another cache
    ca_context* ctx_ = nullptr;
    bool valid_ = false;
    int64_t planned_version_ = -1, planned_appended_ = 0;  // of the tree, at the last refresh
    HostTimes host_times_;

    // The work list of the current tree, shared by the caches made from one another with
    // Attention(other) (a model's layers): whoever refreshes first after a tree change plans, the
    // others find their chunk list identical and only upload.
    struct SharedPlan {
        std::vector<ca_chunk_info> infos;
        int n_seqs = -1;
        ca_plan* plan = nullptr;
        int64_t builds = 0, reuses = 0;
        ~SharedPlan();
    };
    std::shared_ptr<SharedPlan> shared_plan_;

    // The device tables of the current portions (extend), shared the same way: equal tables are uploaded once.
    struct WindowTables {
        torch::Tensor device;  // src_row [rows] | base [entries + 1] | first [entries]
        int64_t rows = 0, pairs = 0;
    };
    struct SharedTables {
        std::vector<int32_t> data;
        torch::Tensor device;
        // made from the portions on demand, by block size and by window
        std::map<int, std::pair<torch::Tensor, int>> blocks;
        std::map<int, WindowTables> windows;
    };
    std::shared_ptr<SharedTables> shared_tables_;
    struct Tables {
        torch::Tensor device;      // tok_slot | path_off | path_chunks | blocks | starts
        int64_t n_tokens = -1, path_off = 0, path_chunks = 0, blocks = 0;
        int n_blocks = 0, block_rows = 1;
        std::vector<int> starts, lens;  // first position and tokens of every entry
    };
    std::shared_ptr<Tables> tables_;
    const std::pair<torch::Tensor, int>& blocks_of(int block_rows);
    const WindowTables& window_tables();
    void need_latent(const char* what) const;
    void need_owner() const;

    // add_seq_async: one worker thread, started on first use, runs the queued insertions in order
    void worker_loop();
    std::thread worker_;
    std::mutex worker_mutex_;
    std::condition_variable worker_cv_;
    std::deque<std::function<void()>> worker_queue_;
    bool worker_stop_ = false;
};

}  // namespace ca_host

// Sequencing shared by the model families (engine_core.h): decode steps replayed as CUDA graphs, the greedy loop, chunked
// prefill, sequence lengths, KV blocks and sampling. The per-token order mirrors TenzoEngineImpl of the reference
// (src/runtime/TenzoEngine.cpp:1809-1838): embedding -> layers -> (generate only) logits + sampler, with the sequence
// length advanced once per token after all layers.
#include "engine_core.h"

#include <nvtx3/nvToolsExt.h>

#include <cmath>
#include <cstdlib>
#include <cstring>

#include "sampler.h"

namespace tz {

thread_local std::string g_last_error;
void set_error(const std::string& m) { g_last_error = m; }

__global__ void advance_kernel(int* pos, int* tokens, const int* next, int batch, int feed_back, int vocab) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < batch) {
        pos[i] += 1;
        if (feed_back) {
            const int t = next[i];
            tokens[i] = (t >= 0 && t < vocab) ? t : 0;
        }
    }
}

__global__ void record_tokens_kernel(const int* next, int* history, int step, int batch) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < batch) history[(size_t)step * batch + i] = next[i];
}

int env_flag(const char* name, int dflt) {
    const char* s = std::getenv(name);
    return s ? std::atoi(s) : dflt;
}

NvtxRange::NvtxRange(const char* name) : on(env_flag("TENZO_NVTX", 0) != 0) { if (on) nvtxRangePushA(name); }
NvtxRange::~NvtxRange() { if (on) nvtxRangePop(); }

void EngineCore::init_core(int b, int graph, int pdl) {
    batch = b > 0 ? b : 1;
    use_graph = graph >= 0 ? graph : env_flag("TENZO_CUDA_GRAPH", 1);
    use_pdl = pdl >= 0 ? pdl : env_flag("TENZO_CUDA_PDL", 1);
    TZ_CUDA(cudaGetDevice(&device));
    TZ_CUDA(cudaStreamCreateWithFlags(&stream, cudaStreamNonBlocking));
    TZ_CUDA(cudaEventCreate(&ev0));
    TZ_CUDA(cudaEventCreate(&ev1));
}

void EngineCore::init_core_buffers() {
    const size_t B = batch;
    d_tokens = (int*)dalloc(B * 4);
    d_pos = (int*)dalloc(B * 4);
    d_next = (int*)dalloc(B * 4);
    b_logits = (float*)dalloc(B * V * 4);
    TZ_CUDA(cudaMallocHost(&h_pin, (3 * B + 16) * sizeof(int)));
    h_tokens = h_pin;
    h_pos = h_pin + B;
    h_next = h_pin + 2 * B;
    seq_len.assign(batch, 0);
}

void* EngineCore::dalloc(size_t bytes) {
    void* p = nullptr;
    TZ_CUDA(cudaMalloc(&p, bytes ? bytes : 16));
    owned.push_back(p);
    TZ_CUDA(cudaMemsetAsync(p, 0, bytes ? bytes : 16, stream));
    return p;
}

// Everything the engine owns, safe to call on a partly constructed object and more than once.
void EngineCore::release_core() {
    if (stream) cudaStreamSynchronize(stream);
    for (auto& kv : graphs) cudaGraphExecDestroy(kv.second);
    graphs.clear();
    for (void* p : owned) cudaFree(p);
    owned.clear();
    if (h_pin) cudaFreeHost(h_pin);
    if (h_table) cudaFreeHost(h_table);
    if (h_cand) cudaFreeHost(h_cand);
    h_pin = nullptr; h_table = nullptr; h_cand = nullptr;
    if (d_sample_past) cudaFree(d_sample_past);
    if (d_history) cudaFree(d_history);
    d_sample_past = nullptr; d_history = nullptr;
    if (ev0) cudaEventDestroy(ev0);
    if (ev1) cudaEventDestroy(ev1);
    if (stream) cudaStreamDestroy(stream);
    ev0 = ev1 = nullptr;
    stream = nullptr;
}

EngineCore::~EngineCore() { release_core(); }

void EngineCore::reserve_blocks(int s, int len) {
    if (!paged) return;
    while (n_blocks[s] * kBlock < len) {
        if (free_blocks.empty()) throw std::out_of_range("the KV block pool is exhausted");   // the reference would reuse block 0 (:302)
        h_table[(size_t)s * table_stride + n_blocks[s]] = free_blocks.back();   // TenzoEngine.h:136-141
        free_blocks.pop_back();
        n_blocks[s] += 1;
        table_dirty = true;
    }
}

void EngineCore::release_blocks(int s, int len) {
    if (!paged) return;
    const int keep = (len + kBlock - 1) / kBlock;
    if (n_blocks[s] <= keep) return;
    TZ_CUDA(cudaStreamSynchronize(stream));               // no step in flight may still read the entries given back
    while (n_blocks[s] > keep) {
        n_blocks[s] -= 1;
        free_blocks.push_back(h_table[(size_t)s * table_stride + n_blocks[s]]);   // TenzoEngine.h:143-147
    }
}

// Entries are only ever added between two synchronising calls (reset_kv, release_blocks), so a copy still queued
// behind earlier steps may carry newer entries without harm: those steps do not read them.
void EngineCore::prepare_kv(int extra) {
    if (!paged) return;
    for (int s = 0; s < batch; ++s) reserve_blocks(s, seq_len[s] + extra);
    if (table_dirty) {
        TZ_CUDA(cudaMemcpyAsync(d_table, h_table, (size_t)batch * table_stride * sizeof(int), cudaMemcpyHostToDevice, stream));
        table_dirty = false;
    }
}

void EngineCore::reset_kv() {                                  // TenzoEngine.cpp:242-246
    for (auto& n : seq_len) n = 0;
    if (!paged) return;
    TZ_CUDA(cudaStreamSynchronize(stream));
    free_blocks.clear();
    for (int i = total_blocks - 1; i >= 0; --i) free_blocks.push_back(i);
    n_blocks.assign(batch, 0);
}

void EngineCore::reset_seq(int s) { set_seq_len(s, 0); }

void EngineCore::set_seq_len(int s, int len) {
    release_blocks(s, len);                    // block pools: the table follows the length
    reserve_blocks(s, len);
    seq_len[s] = len;
}

void EngineCore::kv_fill(int, unsigned long long) { throw std::invalid_argument("this model keeps more than a KV cache: feed it tokens instead"); }

void* EngineCore::upload(const void* host, size_t bytes) {
    void* p = nullptr;
    TZ_CUDA(cudaMalloc(&p, bytes));
    owned.push_back(p);
    TZ_CUDA(cudaMemcpy(p, host, bytes, cudaMemcpyHostToDevice));
    return p;
}

void EngineCore::invalidate_graphs() {
    if (graphs.empty()) return;
    cudaStreamSynchronize(stream);
    for (auto& kv : graphs) cudaGraphExecDestroy(kv.second);
    graphs.clear();
}

int bucket_for(int len, int max_seq) {
    int b = 256;
    while (b < len) b <<= 1;
    return b < max_seq ? b : max_seq;
}

// One step for all sequences. The graph key is (with_logits, feed_back, attention bucket).
void EngineCore::run_step(bool with_logits, bool feed_back) {
    int longest = 0;
    for (int s = 0; s < batch; ++s) {
        if (seq_len[s] + 1 > cfg.max_seq_len) throw std::out_of_range("KV cache is full (max_seq_len reached)");
        longest = seq_len[s] + 1 > longest ? seq_len[s] + 1 : longest;
    }
    const int max_len = step_bucket(longest);
    prepare_kv(1);
    if (direct_step(with_logits, feed_back, max_len, longest)) {
    } else if (!use_graph) {
        enqueue_step(with_logits, feed_back, max_len);
    } else {
        const int key = (with_logits ? 1 : 0) | (feed_back ? 2 : 0) | (max_len << 2);
        auto it = graphs.find(key);
        if (it == graphs.end()) {
            const unsigned long long before = launches;
            cudaGraph_t graph = nullptr;
            TZ_CUDA(cudaStreamBeginCapture(stream, cudaStreamCaptureModeThreadLocal));
            try {
                enqueue_step(with_logits, feed_back, max_len);
            } catch (...) {
                cudaStreamEndCapture(stream, &graph);
                if (graph) cudaGraphDestroy(graph);
                launches = before;
                throw;
            }
            TZ_CUDA(cudaStreamEndCapture(stream, &graph));
            cudaGraphExec_t exec = nullptr;
            cudaError_t e = cudaGraphInstantiate(&exec, graph, 0);
            cudaGraphDestroy(graph);
            if (e != cudaSuccess) throw CudaError(e, "cudaGraphInstantiate");
            graph_kernels[key] = launches - before;
            launches = before;
            it = graphs.emplace(key, exec).first;
        }
        TZ_CUDA(cudaGraphLaunch(it->second, stream));
        launches += graph_kernels[key];
    }
    for (int s = 0; s < batch; ++s) seq_len[s] += 1;   // :1831-1835, once per token
}

void EngineCore::push_state(const int* tokens) {
    for (int s = 0; s < batch; ++s) {
        if (tokens) {
            if (tokens[s] < 0 || tokens[s] >= V) throw std::out_of_range("token id outside [0, vocab_size)");
            h_tokens[s] = tokens[s];
        }
        h_pos[s] = seq_len[s];
    }
    if (tokens) TZ_CUDA(cudaMemcpyAsync(d_tokens, h_tokens, (size_t)batch * 4, cudaMemcpyHostToDevice, stream));
    TZ_CUDA(cudaMemcpyAsync(d_pos, h_pos, (size_t)batch * 4, cudaMemcpyHostToDevice, stream));
}

void EngineCore::enqueue_advance(bool feed_back) {
    advance_kernel<<<(batch + 127) / 128, 128, 0, stream>>>(d_pos, d_tokens, d_next, batch, feed_back ? 1 : 0, V);
    TZ_CUDA(cudaGetLastError());
    launches += 1;
}

void EngineCore::check_tokens(const int* tokens, int n) const {
    for (int i = 0; i < n; ++i)
        if (tokens[i] < 0 || tokens[i] >= V) throw std::out_of_range("token id outside [0, vocab_size)");
}

void EngineCore::prefill_chunk(const int* tokens, int n) {
    NvtxRange range("tenzo.prefill_chunk");
    if (batch != 1) throw std::invalid_argument("chunked prefill is for single-sequence engines");
    if (n > 0) forward(0, tokens, n, nullptr, 0, nullptr);
}

// n consecutive tokens of one sequence; the logits of the rows in `want` (ascending places among them) go to the host.
// A single token of a single-sequence engine is an ordinary decode step, more go through the layers together.
void EngineCore::forward(int s, const int* tokens, int n, const int* want, int n_want, float* logits) {
    if (s < 0 || s >= batch) throw std::out_of_range("sequence index out of range");
    if (n <= 0) throw std::invalid_argument("a portion needs at least one token");
    if (seq_len[s] + n > cfg.max_seq_len) throw std::out_of_range("KV cache is full (max_seq_len reached)");
    check_tokens(tokens, n);
    for (int i = 0; i < n_want; ++i)
        if (want[i] < 0 || want[i] >= n || (i > 0 && want[i] <= want[i - 1])) throw std::out_of_range("wanted rows must ascend inside the portion");
    if (n == 1 && batch == 1) {
        push_state(tokens);
        TZ_CUDA(cudaEventRecord(ev0, stream));
        run_step(n_want > 0, false);
        TZ_CUDA(cudaEventRecord(ev1, stream));
        if (n_want) TZ_CUDA(cudaMemcpyAsync(logits, b_logits, (size_t)V * 4, cudaMemcpyDeviceToHost, stream));
        TZ_CUDA(cudaStreamSynchronize(stream));
        after_sync();
    } else {
        // rows are bounded by kMaxChunkRows, so a long prompt goes through in several portions
        constexpr int kMaxChunkRows = 4096;
        TZ_CUDA(cudaEventRecord(ev0, stream));
        int w = 0;
        for (int a = 0; a < n; a += kMaxChunkRows) {
            const int m = n - a < kMaxChunkRows ? n - a : kMaxChunkRows;
            chunk_rows(s, tokens + a, m);
            std::vector<int> rows;
            for (; w < n_want && want[w] < a + m; ++w) rows.push_back(want[w] - a);
            if (!rows.empty()) rows_logits(rows.data(), (int)rows.size(), logits + (size_t)(w - (int)rows.size()) * V);
        }
        TZ_CUDA(cudaEventRecord(ev1, stream));
        TZ_CUDA(cudaStreamSynchronize(stream));
    }
    check_device_status(false);
}

void EngineCore::prefill(const int* tokens) {
    NvtxRange range("tenzo.prefill_token");
    push_state(tokens);
    TZ_CUDA(cudaEventRecord(ev0, stream));
    run_step(false, false);
    TZ_CUDA(cudaEventRecord(ev1, stream));
    TZ_CUDA(cudaStreamSynchronize(stream));
    after_sync();
}

void EngineCore::generate(const int* cur, int* out) {
    NvtxRange range("tenzo.generate_step");
    push_state(cur);
    TZ_CUDA(cudaEventRecord(ev0, stream));
    run_step(true, false);
    TZ_CUDA(cudaEventRecord(ev1, stream));
    TZ_CUDA(cudaMemcpyAsync(h_next, d_next, (size_t)batch * 4, cudaMemcpyDeviceToHost, stream));
    TZ_CUDA(cudaStreamSynchronize(stream));
    check_device_status(false);
    for (int s = 0; s < batch; ++s) out[s] = h_next[s];
}

void EngineCore::decode_greedy(const int* first, int n_steps, int* out) {
    NvtxRange range("tenzo.decode_greedy");
    if (n_steps <= 0) return;
    if ((size_t)n_steps * batch > history_cap) {
        if (d_history) cudaFree(d_history);
        d_history = nullptr;
        TZ_CUDA(cudaMalloc((void**)&d_history, (size_t)n_steps * batch * 4));
        history_cap = (size_t)n_steps * batch;
    }
    push_state(first);
    TZ_CUDA(cudaEventRecord(ev0, stream));
    for (int i = 0; i < n_steps; ++i) {
        run_step(true, true);
        record_tokens_kernel<<<(batch + 127) / 128, 128, 0, stream>>>(d_next, d_history, i, batch);
        launches += 1;
    }
    TZ_CUDA(cudaEventRecord(ev1, stream));
    TZ_CUDA(cudaMemcpyAsync(out, d_history, (size_t)n_steps * batch * 4, cudaMemcpyDeviceToHost, stream));
    TZ_CUDA(cudaStreamSynchronize(stream));
    after_sync();
    check_device_status(true);
}

float EngineCore::last_ms() {
    float ms = 0.0f;
    if (cudaEventElapsedTime(&ms, ev0, ev1) != cudaSuccess) return -1.0f;
    return ms;
}

// The reference sampler (TenzoEngine.cpp:1722-1807) on host logits, for the stochastic path and
// for greedy decoding with a repetition penalty. Candidate order follows std::pair<float,int>.
// The reference's streaming top-k, softmax, top-p and draw (TenzoEngine.cpp:1745-1806) over pairs in ascending index order.
int sample_pairs(const float* vals, const int* idxs, int n_in, const tenzo_sampling_params_t& p, float r_in) {
    if (n_in <= 0) return 0;
    if (p.temperature <= 0.0f) {                          // first maximum (:1746-1755)
        int best = 0;
        for (int i = 1; i < n_in; ++i)
            if (vals[i] > vals[best]) best = i;
        return idxs ? idxs[best] : best;
    }
    const int top_k = p.top_k < 1 ? 1 : (p.top_k > 64 ? 64 : p.top_k);
    float cl[64];
    int ci[64], n = 0;
    for (int j = 0; j < n_in; ++j) {                      // sorted insert = the min-heap of (value, index) pairs, :1760-1768
        const float l = vals[j];
        const int i = idxs ? idxs[j] : j;
        if (n == top_k) {
            if (!(l > cl[n - 1])) continue;
            --n;
        }
        int q = n;
        while (q > 0 && (cl[q - 1] < l || (!(l < cl[q - 1]) && ci[q - 1] < i))) { cl[q] = cl[q - 1]; ci[q] = ci[q - 1]; --q; }
        cl[q] = l; ci[q] = i; ++n;
    }
    float probs[64], sum = 0.0f;
    for (int i = 0; i < n; ++i) { probs[i] = std::exp((cl[i] - cl[0]) / p.temperature); sum += probs[i]; }
    for (int i = 0; i < n; ++i) probs[i] /= sum;
    float cum = 0.0f;
    int cut = n;
    for (int i = 0; i < n; ++i) { cum += probs[i]; if (cum >= p.top_p) { cut = i + 1; break; } }
    float sub = 0.0f;
    for (int i = 0; i < cut; ++i) sub += probs[i];
    for (int i = 0; i < cut; ++i) probs[i] /= sub;
    const float r = r_in >= 0.0f ? r_in : static_cast<float>(std::rand()) / static_cast<float>(RAND_MAX);   // :1800, process-global rand()
    float acc = 0.0f;
    for (int i = 0; i < cut; ++i) { acc += probs[i]; if (r <= acc) return ci[i]; }
    return ci[0];
}

// Penalty, k-th-largest selection and candidate compaction on the device (sampler.cu), the rest on the host.
int EngineCore::sample(const tenzo_sampling_params_t& p, const int* past, int n_past) {
    if (batch != 1) throw std::invalid_argument("sampling with parameters is per sequence");
    if (p.repetition_penalty != 1.0f && past && n_past > 0) {
        std::map<int, int> mult;                          // once per occurrence (:1736-1742)
        for (int i = 0; i < n_past; ++i) ++mult[past[i]];
        std::vector<int> toks, cnts;
        for (auto& kv : mult) { toks.push_back(kv.first); cnts.push_back(kv.second); }
        const size_t n = toks.size();
        if (n > sample_past_cap) {
            if (d_sample_past) cudaFree(d_sample_past);
            sample_past_cap = n * 2;
            TZ_CUDA(cudaMalloc((void**)&d_sample_past, sample_past_cap * 2 * sizeof(int)));
        }
        TZ_CUDA(cudaMemcpyAsync(d_sample_past, toks.data(), n * 4, cudaMemcpyHostToDevice, stream));
        TZ_CUDA(cudaMemcpyAsync(d_sample_past + sample_past_cap, cnts.data(), n * 4, cudaMemcpyHostToDevice, stream));
        TZ_CUDA(launch_penalty(b_logits, V, d_sample_past, d_sample_past + sample_past_cap, (int)n, p.repetition_penalty, stream));
        launches += 1;
    }
    const int k = p.temperature <= 0.0f ? 1 : (p.top_k < 1 ? 1 : (p.top_k > 64 ? 64 : p.top_k));
    if (!d_cand) {
        TZ_CUDA(cudaMalloc((void**)&d_cand, 16 + (size_t)kMaxCandidates * 8));
        owned.push_back(d_cand);
        TZ_CUDA(cudaMallocHost((void**)&h_cand, 16 + (size_t)kMaxCandidates * 8));
    }
    int* d_count = reinterpret_cast<int*>(d_cand);
    float* d_val = reinterpret_cast<float*>(static_cast<unsigned char*>(d_cand) + 16);
    int* d_idx = reinterpret_cast<int*>(d_val + kMaxCandidates);
    TZ_CUDA(launch_select_candidates(b_logits, V, k, d_count, d_val, d_idx, stream));
    launches += 1;
    TZ_CUDA(cudaMemcpyAsync(h_cand, d_cand, 16 + (size_t)kMaxCandidates * 8, cudaMemcpyDeviceToHost, stream));
    TZ_CUDA(cudaStreamSynchronize(stream));
    const int count = *reinterpret_cast<const int*>(h_cand);
    const float* hv = reinterpret_cast<const float*>(static_cast<unsigned char*>(h_cand) + 16);
    const int* hi = reinterpret_cast<const int*>(hv + kMaxCandidates);
    if (count > kMaxCandidates) {                         // a huge tie at the threshold: take the whole vector
        std::vector<float> lg((size_t)V);
        TZ_CUDA(cudaMemcpy(lg.data(), b_logits, lg.size() * 4, cudaMemcpyDeviceToHost));
        return sample_pairs(lg.data(), nullptr, V, p, -1.0f);
    }
    return sample_pairs(hv, hi, count, p, -1.0f);
}

}  // namespace tz

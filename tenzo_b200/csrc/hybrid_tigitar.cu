// Tigitar on the hybrid decoders (hybrid_engine.h): its configuration and weights as HybridLayer entries. Norms stand in front
// of and behind every sublayer; mixers are the gated delta rule and sliding-window attention over latents, whose cache a
// later layer may borrow; feed-forwards are dense ReLU GLUs or mixtures of SiLU GLU experts; logits are soft-capped.
#include <algorithm>
#include <cmath>

#include "hybrid_engine.h"

namespace tz {

// No position is learned, so the length of a sequence is bounded by nothing but this.
constexpr int kTigitarPositions = 1 << 20;

static int positive(const Json& j, const char* key) {
    const int v = j.at(key).integer();
    if (v < 1) throw std::invalid_argument(std::string("'") + key + "' has to be positive");
    return v;
}
static int head_size(const Json& j, const char* key) {
    const int v = positive(j, key);
    if (v > kMaxHeadDim) throw std::invalid_argument(std::string("'") + key + "' is limited to " + std::to_string(kMaxHeadDim));
    return v;
}

void HybridEngine::read_delta(HybridLayer& y, const Json& mix, const SafeTensors& st, const std::string& pre) {
    y.has_delta = true;
    DeltaMixer& m = y.delta;
    m.heads = positive(mix, "heads");
    m.kv_heads = positive(mix, "kv_heads");
    m.dim = head_size(mix, "dim");
    m.vdim = head_size(mix, "vdim");
    m.taps = positive(mix, "conv");
    if (m.heads % m.kv_heads) throw std::invalid_argument("heads must be a multiple of kv_heads");
    if (m.taps > kMaxTaps) throw std::invalid_argument("'conv' is limited to " + std::to_string(kMaxTaps));
    const int nk = m.kv_heads * m.dim, nv = m.heads * m.vdim;
    m.conv_q = conv_weights(st, pre + "q.conv", nk, m.taps);
    m.conv_k = conv_weights(st, pre + "k.conv", nk, m.taps);
    m.conv_v = conv_weights(st, pre + "v.conv", nv, m.taps);
    m.a_log = upload_floats(st.floats(pre + "A_log", {m.heads}));
    m.dt_bias = upload_floats(st.floats(pre + "dt_bias", {m.heads}));
    m.norm = upload_floats(st.floats(pre + "norm", {m.vdim}));
    m.state = take_state((size_t)m.heads * m.dim * round_up(m.vdim, 4));
    m.tail = take_state((size_t)m.taps * m.channels());
    m.o = make_weight(h, nv);
    upload_weight(m.o, 0, st, pre + "o", h, nv);
    fuse_inputs(y, {{pre + "q", nk, &m.off_q}, {pre + "k", nk, &m.off_k}, {pre + "v", nv, &m.off_v}, {pre + "g", nv, &m.off_g},
                    {pre + "a", m.heads, &m.off_a}, {pre + "b", m.heads, &m.off_b}}, 8, st);
}

// cache_of[l]: the cache that layer l makes, -1 for none.
void HybridEngine::read_latent(int l, const Json& config, const SafeTensors& st, const std::string& pre, std::vector<int>& cache_of) {
    HybridLayer& y = layers[l];
    const Json& mix = config.at("layers").array()[l].at("mixer");
    y.has_latent = true;
    LatentMixer& m = y.lat;
    m.heads = positive(mix, "heads");
    m.dim = head_size(mix, "dim");
    m.vdim = head_size(mix, "vdim");
    m.window = positive(mix.at("mask"), "size");
    m.scale = (float)mix.at("scale").number();
    const int rank = positive(mix, "kv_rank"), rot = head_size(mix, "rot_dim");
    if (rank > kMaxLatentRank) throw std::invalid_argument("'kv_rank' is limited to " + std::to_string(kMaxLatentRank));
    if (rot % 2 || mix.at("rot").at("dims").integer() != rot) throw std::invalid_argument("the rotated part has to be even and rotated as a whole");
    std::vector<double> freq(rot / 2);
    for (int i = 0; i < rot / 2; ++i) freq[i] = std::pow(mix.at("rot").at("base").number(), -2.0 * i / rot);
    const int ring = std::min(m.window, n_pos);

    std::vector<Piece> pieces = {{pre + "q", m.heads * (m.dim + rot), &m.off_q}};
    m.owner = !mix.has("kv_from") || mix.at("kv_from").is_null();
    if (m.owner) {
        LatentCache k;
        k.rank = rank;
        k.rot = rot;
        k.ring = ring;
        k.freq = (double*)upload(freq.data(), freq.size() * sizeof(double));
        m.cache = cache_of[l] = (int)caches.size();
        caches.push_back(k);
        m.norm = upload_floats(st.floats(pre + "dkv.norm", {rank}));
        pieces.push_back({pre + "dkv", rank + rot, &m.off_dkv});
    } else {
        const int from = mix.at("kv_from").integer();
        if (from < 0 || from >= l || cache_of[from] < 0) throw std::invalid_argument("'kv_from' has to name an earlier layer with a latent of its own");
        m.cache = cache_of[from];
        LatentCache& k = caches[m.cache];
        const Json& other = config.at("layers").array()[from].at("mixer").at("rot");
        if (k.rank != rank || k.rot != rot || other.at("base").number() != mix.at("rot").at("base").number())
            throw std::invalid_argument("a layer and the one named by 'kv_from' need the same kv_rank, rot_dim and rotation");
        k.borrowed = true;
        k.ring = std::max(k.ring, ring);
    }
    const int ld = round_up(rank, 64), d8 = m.dim8(), v8 = m.vdim8();
    m.kv = (bf16*)dalloc((size_t)m.heads * (d8 + v8) * ld * 2);
    TZ_CUDA(cudaStreamSynchronize(stream));                // zeroed before the copies below
    const TensorView &uk = st.bf16(pre + "uk", {m.heads * m.dim, rank}), &uv = st.bf16(pre + "uv", {m.heads * m.vdim, rank});
    for (int i = 0; i < m.heads; ++i) {
        TZ_CUDA(cudaMemcpy2DAsync(m.kv + (size_t)i * d8 * ld, (size_t)ld * 2, uk.data + (size_t)i * m.dim * rank * 2, (size_t)rank * 2, (size_t)rank * 2,
                                  (size_t)m.dim, cudaMemcpyHostToDevice, stream));
        TZ_CUDA(cudaMemcpy2DAsync(m.kv + ((size_t)m.heads * d8 + (size_t)i * v8) * ld, (size_t)ld * 2, uv.data + (size_t)i * m.vdim * rank * 2, (size_t)rank * 2,
                                  (size_t)rank * 2, (size_t)m.vdim, cudaMemcpyHostToDevice, stream));
    }
    m.o = make_weight(h, m.heads * v8);
    const TensorView& o = st.bf16(pre + "o", {h, m.heads * m.vdim});
    for (int i = 0; i < m.heads; ++i)
        TZ_CUDA(cudaMemcpy2DAsync(m.o.w + (size_t)i * v8, (size_t)m.o.ld_k * 2, o.data + (size_t)i * m.vdim * 2, (size_t)m.heads * m.vdim * 2, (size_t)m.vdim * 2,
                                  (size_t)h, cudaMemcpyHostToDevice, stream));
    TZ_CUDA(cudaStreamSynchronize(stream));
    fuse_inputs(y, pieces, 8, st);
}

// Matrices `index` of up (2 ff rows, gate and up interleaved) and down (as many rows as the model is wide).
void HybridEngine::read_glu(DenseWeight& up, DenseWeight& down, int index, int ff, const SafeTensors& st, const std::string& pre) {
    for (int i = 0; i < 2; ++i) {
        const TensorView& t = st.bf16(pre + (i ? "up" : "gate"), {ff, h});
        TZ_CUDA(cudaMemcpy2DAsync(up.w + ((size_t)index * 2 * ff + i) * up.ld_k, (size_t)up.ld_k * 4, t.data, (size_t)h * 2, (size_t)h * 2, (size_t)ff,
                                  cudaMemcpyHostToDevice, stream));
    }
    upload_weight(down, index * h, st, pre + "down", h, ff);
}

void HybridEngine::load_tigitar(const Json& c, const SafeTensors& st) {
    h = positive(c, "width");
    V = positive(c, "vocab");
    n_pos = kTigitarPositions;
    eps = (float)c.at("norm").at("eps").number();
    if (c.has("logit_softcap") && !c.at("logit_softcap").is_null()) {
        logit_cap = (float)c.at("logit_softcap").number();
        if (!(logit_cap > 0.0f)) throw std::invalid_argument("'logit_softcap' has to be positive");
    }
    const auto& list = c.at("layers").array();
    start_layers((int)list.size());
    embed = (bf16*)upload(st.bf16("embed", {V, h}).data, (size_t)V * h * 2);
    final_gain_w = upload_floats(st.floats("final.norm", {h}));
    head = make_weight(V, h);
    upload_weight(head, 0, st, "head", V, h);

    std::vector<int> cache_of(L, -1);
    for (int l = 0; l < L; ++l) {
        HybridLayer& y = layers[l];
        const std::string p = "l" + std::to_string(l) + ".", type = list[l].at("type").string();
        auto norm = [&](const char* name) { return upload_floats(st.floats(p + name, {h})); };
        y.norm1_w = norm("norm1");
        y.post1_w = norm("norm1b");
        if (type == "delta") read_delta(y, list[l].at("mixer"), st, p + "mix.");
        else if (type == "latent_attention") read_latent(l, c, st, p + "mix.", cache_of);
        else throw std::invalid_argument("layer " + std::to_string(l) + ": unknown type '" + type + "'");

        const Json& mlp = list[l].at("mlp");
        if (mlp.is_null()) continue;
        y.has_mlp = true;
        y.norm2_w = norm("norm2");
        y.post2_w = norm("norm2b");
        const std::string kind = mlp.at("kind").string(), mp = p + "mlp.";
        if (kind == "dense") {
            const int ff = positive(mlp, "ff");
            y.up = make_weight(2 * ff, h);
            y.down = make_weight(h, ff);
            y.up_epilogue = TENZO_GEMM_GLU_RELU;
            read_glu(y.up, y.down, 0, ff, st, mp);
        } else if (kind == "moe") {
            ExpertMlp& m = y.moe;
            m.experts = positive(mlp.at("router"), "experts");
            m.top = positive(mlp.at("router"), "top");
            m.ff = positive(mlp.at("expert"), "ff");
            if (m.top > m.experts) throw std::invalid_argument("layer " + std::to_string(l) + ": more experts per token than there are");
            m.router = make_weight(m.experts, h);
            upload_weight(m.router, 0, st, mp + "router", m.experts, h);
            m.correction = upload_floats(st.floats(mp + "correction", {m.experts}));
            m.up = make_weight(m.experts * 2 * m.ff, h);
            m.down = make_weight(m.experts * h, m.ff);
            for (int e = 0; e < m.experts; ++e) read_glu(m.up, m.down, e, m.ff, st, mp + "e" + std::to_string(e) + ".");
        } else {
            throw std::invalid_argument("layer " + std::to_string(l) + ": unknown feed-forward '" + kind + "'");
        }
    }
}

static EngineCore* open_tigitar(const Json& config, const OpenOptions& o) { return new HybridEngine(config, o, &HybridEngine::load_tigitar); }
static const ModelRegistration registration({"Tigitar", open_tigitar});

}  // namespace tz

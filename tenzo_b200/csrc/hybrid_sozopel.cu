// Sozopel on the hybrid decoders (hybrid_engine.h): its configuration and weights as HybridLayer entries.
#include <algorithm>
#include <cmath>

#include "hybrid_engine.h"

namespace tz {

static double softplus(double z) { return std::max(z, 0.0) + std::log1p(std::exp(-std::fabs(z))); }

void HybridEngine::read_window(WindowMixer& m, const Json& mix) {
    m.heads = mix.at("heads").integer();
    m.kv_heads = mix.at("kv_heads").integer();
    m.dim = mix.at("dim").integer();
    m.vdim = mix.at("vdim").integer();
    m.taps = mix.at("conv").integer();
    m.window = mix.at("mask").at("size").integer();
    m.scale = (float)mix.at("scale").number();
    if (m.heads < 1 || m.kv_heads < 1 || m.heads % m.kv_heads) throw std::invalid_argument("heads must be a multiple of kv_heads");
    if (m.dim < 1 || m.dim > kMaxHeadDim || m.vdim < 1 || m.vdim > kMaxHeadDim) throw std::invalid_argument("attention head sizes are limited to 256");
    if (m.taps < 1 || m.taps > kMaxTaps || m.window < 1) throw std::invalid_argument("bad convolution or window size");
    m.ring = std::min(m.window, n_pos);
}

static void read_scan(ScanMixer& m, const Json& mix, bool square) {
    m.heads = mix.at("heads").integer();
    m.dim = mix.at("dim").integer();
    m.vdim = square ? m.dim : mix.at("vdim").integer();
    if (m.heads < 1 || m.dim < 1 || m.dim > kMaxHeadDim || m.vdim < 1 || m.vdim > kMaxHeadDim)
        throw std::invalid_argument("recurrent head sizes are limited to 256");
}

void HybridEngine::load_sozopel(const Json& c, const SafeTensors& st) {
    h = c.at("width").integer();
    V = c.at("vocab").integer();
    n_pos = c.at("max_positions").integer();
    eps = (float)c.at("norm").at("eps").number();
    taps = c.at("canon").at("taps").integer();
    if (taps < 1 || taps > kMaxTaps) throw std::invalid_argument("canon.taps is limited to 1..16");
    start_layers((int)c.at("layers").array().size());
    const int W = h;
    embed = (bf16*)upload(st.bf16("embed", {V, W}).data, (size_t)V * W * 2);
    pos_table = (bf16*)upload(st.bf16("pos", {n_pos, W}).data, (size_t)n_pos * W * 2);
    final_gain = st.floats("final.norm", {})[0];
    head = make_weight(V, W);
    upload_weight(head, 0, st, "head", V, W);

    const auto& list = c.at("layers").array();
    for (int l = 0; l < L; ++l) {
        HybridLayer& y = layers[l];
        const Json& e = list[l];
        const std::string p = "l" + std::to_string(l) + ".", mp = p + "mix.", type = e.at("type").string();
        const Json& mix = e.at("mixer");
        y.norm1 = st.floats(p + "norm1", {})[0];
        y.canon1 = conv_weights(st, p + "canon1", W, taps);
        y.tail1 = take_tail((size_t)(taps - 1) * W);

        // the fused input projection: (tensor, rows, where its column goes), pieces at multiples of `align` columns
        std::vector<Piece> pieces;
        int align = 8;
        auto scan_common = [&](const std::string& pre) {
            ScanMixer& s = y.scan;
            y.has_scan = true;
            s.state = take_state((size_t)s.heads * s.dim * round_up(s.vdim, 4));
            s.o = make_weight(W, s.heads * s.vdim);
            upload_weight(s.o, 0, st, pre + "o", W, s.heads * s.vdim);
        };
        auto low_rank = [&](const std::string& down, const std::string& up_name, const std::string& bias) {
            ScanMixer& s = y.scan;
            s.rank = (int)st.bf16(down, {-1, W}).shape[0];
            const int n = s.heads * s.dim;
            s.up = (bf16*)dalloc((size_t)n * round_up(s.rank, 8) * 2);
            TZ_CUDA(cudaMemcpy2DAsync(s.up, (size_t)round_up(s.rank, 8) * 2, st.bf16(up_name, {n, s.rank}).data, (size_t)s.rank * 2, (size_t)s.rank * 2,
                                      (size_t)n, cudaMemcpyHostToDevice, stream));
            TZ_CUDA(cudaStreamSynchronize(stream));
            s.bias = upload_floats(st.floats(bias, {n}));
        };
        if (type == "retention") {
            ScanMixer& s = y.scan;
            read_scan(s, mix, false);
            s.k_scale = (float)std::pow((double)s.dim, -0.5);
            s.decay_kind = TENZO_DECAY_CONST;
            std::vector<float> d;
            for (const Json& v : mix.at("decay").array()) d.push_back((float)v.number());
            if ((int)d.size() != s.heads) throw std::invalid_argument("'decay' needs one entry per head");
            s.decay = upload_floats(d);
            scan_common(mp);
            pieces = {{mp + "q", s.heads * s.dim, &s.off_q}, {mp + "k", s.heads * s.dim, &s.off_k},
                      {mp + "v", s.heads * s.vdim, &s.off_v}, {mp + "g", s.heads * s.vdim, &s.off_g}};
        } else if (type == "wkv") {
            ScanMixer& s = y.scan;
            read_scan(s, mix, true);
            s.decay_kind = TENZO_DECAY_EXP_EXP;
            low_rank(mp + "w1", mp + "w2", mp + "w0");
            s.bonus = upload_floats(st.floats(mp + "u", {s.heads, s.dim}));
            s.norm = upload_floats(st.floats(mp + "norm", {s.heads * s.vdim}));
            s.norm_per_head = 1;
            scan_common(mp);
            const int n = s.heads * s.dim;
            pieces = {{mp + "r", n, &s.off_q}, {mp + "k", n, &s.off_k}, {mp + "v", n, &s.off_v}, {mp + "g", n, &s.off_g}, {mp + "w1", s.rank, &s.off_low}};
            align = 128;                           // each piece multiplies its own mix: a segment of the product
            y.n_mix = 5;
            std::vector<float> mu;
            for (const char* m : {"r", "k", "v", "g", "w"}) {
                const std::vector<float> v = st.floats(mp + "mu." + m, {W});
                mu.insert(mu.end(), v.begin(), v.end());
            }
            y.mu = upload_floats(mu);
            y.prev = take_tail(W);
        } else if (type == "parallel") {
            WindowMixer& m = y.win;
            y.has_window = true;
            read_window(m, mix.at("left"));
            const std::string lp = mp + "left.", rp = mp + "right.";
            m.conv_q = conv_weights(st, lp + "q.conv", m.heads * m.dim, m.taps);
            m.conv_k = conv_weights(st, lp + "k.conv", m.kv_heads * m.dim, m.taps);
            m.conv_v = conv_weights(st, lp + "v.conv", m.kv_heads * m.vdim, m.taps);
            m.tail = take_tail((size_t)(m.taps - 1) * m.channels());
            m.o = make_weight(W, m.heads * m.vdim);
            upload_weight(m.o, 0, st, lp + "o", W, m.heads * m.vdim);
            ScanMixer& s = y.scan;
            read_scan(s, mix.at("right"), false);
            s.q_scale = (float)std::pow((double)s.dim, -0.5);
            s.decay_kind = TENZO_DECAY_SIGMOID_ROOT;
            s.tau = (float)mix.at("right").at("tau").number();
            low_rank(rp + "a1", rp + "a2", rp + "a2.b");
            s.norm = upload_floats(st.floats(rp + "norm", {s.vdim}));
            scan_common(rp);
            y.left_out = upload_floats(st.floats(lp + "out", {W}));
            y.right_out = upload_floats(st.floats(rp + "out", {W}));
            pieces = {{lp + "q", m.heads * m.dim, &m.off_q}, {lp + "k", m.kv_heads * m.dim, &m.off_k}, {lp + "v", m.kv_heads * m.vdim, &m.off_v},
                      {rp + "q", s.heads * s.dim, &s.off_q}, {rp + "k", s.heads * s.dim, &s.off_k}, {rp + "v", s.heads * s.vdim, &s.off_v},
                      {rp + "g", s.heads * s.vdim, &s.off_g}, {rp + "a1", s.rank, &s.off_low}};
        } else {
            throw std::invalid_argument("layer " + std::to_string(l) + ": unknown type '" + type + "'");
        }
        fuse_inputs(y, pieces, align, st);

        if (!e.at("mlp").is_null()) {
            const Json& mlp = e.at("mlp");
            if (mlp.at("kind").string() != "dense") throw std::invalid_argument("layer " + std::to_string(l) + ": unknown feed-forward '" + mlp.at("kind").string() + "'");
            const int ff = mlp.at("ff").integer();
            if (ff < 1) throw std::invalid_argument("non-positive dimension");
            y.has_mlp = true;
            y.norm2 = st.floats(p + "norm2", {})[0];
            y.canon2 = conv_weights(st, p + "canon2", W, taps);
            y.tail2 = take_tail((size_t)(taps - 1) * W);
            y.up = make_weight(ff, W);
            upload_weight(y.up, 0, st, p + "mlp.up", ff, W);
            y.down = make_weight(W, ff);
            upload_weight(y.down, 0, st, p + "mlp.down", W, ff);
            const std::vector<float> act = st.floats(p + "mlp.act", {2});
            y.act_pos = (float)softplus(act[0]);
            y.act_neg = (float)(0.5 + softplus(act[1]));
        }
    }
}

static EngineCore* open_sozopel(const Json& config, const OpenOptions& o) { return new HybridEngine(config, o, &HybridEngine::load_sozopel); }
static const ModelRegistration registration({"Sozopel", open_sozopel});

}  // namespace tz

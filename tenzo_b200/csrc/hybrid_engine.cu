// Hybrid decoders on the shared engine (hybrid_engine.h): configuration, weights, state and the walk through the layers.
//
// One layer, M rows (decode: one per sequence; chunk: consecutive tokens of one sequence):
//   rows     x += what the previous sublayer left, norm1, convolution (, token-shift mixes)
//   gemm     every projection of the mixer's input in one product
//   window   convolution on q, k, v, ring update, attention          } whichever the mixer has
//   scan     decays, recurrence, per-head norm, gate                  }
//   gemm     output projection(s)
//   rows, gemm (+ activation), gemm    the feed-forward, when the layer has one
// Residual sums happen at the start of the next row kernel.
#include "hybrid_engine.h"

#include <algorithm>
#include <cmath>
#include <cstring>

namespace tz {

static double softplus(double z) { return std::max(z, 0.0) + std::log1p(std::exp(-std::fabs(z))); }

HybridEngine::HybridEngine(const Json& config, const OpenOptions& o) {
    try {
        init(config, o);
    } catch (...) {
        free_rows(dec);
        free_rows(chunk);
        release_core();
        throw;
    }
}

HybridEngine::~HybridEngine() {
    if (stream) cudaStreamSynchronize(stream);
    free_rows(dec);
    free_rows(chunk);
}

void HybridEngine::init(const Json& c, const OpenOptions& o) {
    f32 = o.compute == TENZO_COMPUTE_F32;
    h = c.at("width").integer();
    V = c.at("vocab").integer();
    n_pos = c.at("max_positions").integer();
    L = (int)c.at("layers").array().size();
    eps = (float)c.at("norm").at("eps").number();
    taps = c.at("canon").at("taps").integer();
    if (h <= 0 || V <= 0 || n_pos <= 0 || L <= 0) throw std::invalid_argument("non-positive dimension");
    if (taps < 1 || taps > kMaxTaps) throw std::invalid_argument("canon.taps is limited to 1..16");
    cfg = {};
    cfg.hidden_size = h;
    cfg.vocab_size = V;
    cfg.num_layers = L;
    cfg.max_seq_len = n_pos;
    cfg.kv_mode = f32 ? "window_f32" : "window_bf16";
    cfg.device = "cuda";
    init_core(o.opt.batch, o.opt.use_graph, o.opt.use_pdl);
    init_core_buffers();
    load(c, o.dir);

    const size_t B = batch, es = f32 ? 4 : 2;
    tails = (float*)dalloc(B * tail_floats * 4);
    tail_stage = (float*)dalloc(tail_floats * 4);
    states = (float*)dalloc(B * state_floats * 4);
    for (HybridLayer& y : layers) {
        if (!y.has_window) continue;
        WindowMixer& m = y.win;
        m.ring_k_stride = (size_t)m.kv_heads * m.ring * round_up(m.dim, 8);
        m.ring_v_stride = (size_t)m.kv_heads * m.ring * round_up(m.vdim, 8);
        m.ring_k = dalloc(B * m.ring_k_stride * es);
        m.ring_v = dalloc(B * m.ring_v_stride * es);
    }
    gemm_ws = dalloc(tenzo_cuda_gemm_workspace_bytes());
    argmax_ws = dalloc(argmax_scratch_bytes(batch));
    alloc_rows(dec, batch);
    b_x = dec.x;
    TZ_CUDA(cudaStreamSynchronize(stream));
}

// ---- weights --------------------------------------------------------------------------------------------------------------
DenseWeight HybridEngine::make_weight(int rows, int k) {
    DenseWeight d;
    d.rows = rows;
    d.k = k;
    d.ld_k = round_up(k, 64);
    d.w = (bf16*)dalloc((size_t)rows * d.ld_k * 2);
    return d;
}

void HybridEngine::upload_weight(DenseWeight& d, int row0, const SafeTensors& st, const std::string& name, int rows, int k) {
    const TensorView& t = st.bf16(name, {rows, k});
    TZ_CUDA(cudaMemcpy2DAsync(d.w + (size_t)row0 * d.ld_k, (size_t)d.ld_k * 2, t.data, (size_t)k * 2, (size_t)k * 2, (size_t)rows,
                              cudaMemcpyHostToDevice, stream));
    TZ_CUDA(cudaStreamSynchronize(stream));
}

float* HybridEngine::upload_floats(const std::vector<float>& v) { return (float*)upload(v.data(), v.size() * 4); }

float* HybridEngine::conv_weights(const SafeTensors& st, const std::string& name, int channels, int n_taps) {
    const std::vector<float> w = st.floats(name, {channels, n_taps});
    std::vector<float> t(w.size());
    for (int c = 0; c < channels; ++c)
        for (int j = 0; j < n_taps; ++j) t[(size_t)j * channels + c] = w[(size_t)c * n_taps + j];
    return upload_floats(t);
}

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

void HybridEngine::load(const Json& c, const std::string& dir) {
    const SafeTensors st(dir + "/model.safetensors");
    const int W = h;
    embed = (bf16*)upload(st.bf16("embed", {V, W}).data, (size_t)V * W * 2);
    pos_table = (bf16*)upload(st.bf16("pos", {n_pos, W}).data, (size_t)n_pos * W * 2);
    final_gain = st.floats("final.norm", {})[0];
    head = make_weight(V, W);
    upload_weight(head, 0, st, "head", V, W);

    size_t tail = 0, state = 0;
    auto take = [](size_t& at, size_t n) {
        const size_t a = at;
        at += (n + 3) / 4 * 4;                    // 16-byte pieces
        return a;
    };
    max_in = round_up(W, 64);
    const auto& list = c.at("layers").array();
    layers.resize(L);
    for (int l = 0; l < L; ++l) {
        HybridLayer& y = layers[l];
        const Json& e = list[l];
        const std::string p = "l" + std::to_string(l) + ".", mp = p + "mix.", type = e.at("type").string();
        const Json& mix = e.at("mixer");
        y.norm1 = st.floats(p + "norm1", {})[0];
        y.canon1 = conv_weights(st, p + "canon1", W, taps);
        y.tail1 = take(tail, (size_t)(taps - 1) * W);

        // the fused input projection: (tensor, rows, where its column goes), pieces at multiples of `align` columns
        struct Piece { std::string name; int rows; int* off; };
        std::vector<Piece> pieces;
        int align = 8;
        auto scan_common = [&](const std::string& pre) {
            ScanMixer& s = y.scan;
            y.has_scan = true;
            s.state = take(state, (size_t)s.heads * s.dim * round_up(s.vdim, 4));
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
            y.prev = take(tail, W);
        } else if (type == "parallel") {
            WindowMixer& m = y.win;
            y.has_window = true;
            read_window(m, mix.at("left"));
            const std::string lp = mp + "left.", rp = mp + "right.";
            m.conv_q = conv_weights(st, lp + "q.conv", m.heads * m.dim, m.taps);
            m.conv_k = conv_weights(st, lp + "k.conv", m.kv_heads * m.dim, m.taps);
            m.conv_v = conv_weights(st, lp + "v.conv", m.kv_heads * m.vdim, m.taps);
            m.tail = take(tail, (size_t)(m.taps - 1) * m.channels());
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
        int n = 0;
        y.n_seg = 0;
        for (size_t i = 0; i < pieces.size(); ++i) {
            *pieces[i].off = n;
            n += i + 1 < pieces.size() ? round_up(pieces[i].rows, align) : pieces[i].rows;
            if (y.n_mix) y.seg_end[y.n_seg++] = n;
        }
        if (!y.n_mix) y.seg_end[y.n_seg++] = n;
        y.in = make_weight(n, W);
        for (const Piece& q : pieces) upload_weight(y.in, *q.off, st, q.name, q.rows, W);
        max_proj = std::max(max_proj, round_up(n, 8));
        max_seg = std::max(max_seg, std::max(1, y.n_mix));
        if (y.has_window) max_mix = std::max(max_mix, y.win.o.ld_k);
        if (y.has_scan) max_mix = std::max(max_mix, y.scan.o.ld_k);

        if (!e.at("mlp").is_null()) {
            const Json& mlp = e.at("mlp");
            if (mlp.at("kind").string() != "dense") throw std::invalid_argument("layer " + std::to_string(l) + ": unknown feed-forward '" + mlp.at("kind").string() + "'");
            const int ff = mlp.at("ff").integer();
            if (ff < 1) throw std::invalid_argument("non-positive dimension");
            y.has_mlp = true;
            y.norm2 = st.floats(p + "norm2", {})[0];
            y.canon2 = conv_weights(st, p + "canon2", W, taps);
            y.tail2 = take(tail, (size_t)(taps - 1) * W);
            y.up = make_weight(ff, W);
            upload_weight(y.up, 0, st, p + "mlp.up", ff, W);
            y.down = make_weight(W, ff);
            upload_weight(y.down, 0, st, p + "mlp.down", W, ff);
            const std::vector<float> act = st.floats(p + "mlp.act", {2});
            y.act_pos = (float)softplus(act[0]);
            y.act_neg = (float)(0.5 + softplus(act[1]));
            max_ff = std::max(max_ff, y.down.ld_k);
        }
    }
    tail_floats = std::max<size_t>(tail, 4);
    state_floats = std::max<size_t>(state, 4);
}

// ---- activations ------------------------------------------------------------------------------------------------------------
void HybridEngine::free_rows(Rows& r) {
    for (void* p : r.owned) cudaFree(p);
    r = Rows();
}

void HybridEngine::alloc_rows(Rows& r, int cap) {
    free_rows(r);
    const size_t m = cap, es = f32 ? 4 : 2;
    auto get = [&](size_t bytes) -> void* {
        void* p = nullptr;
        TZ_CUDA(cudaMalloc(&p, bytes ? bytes : 16));
        r.owned.push_back(p);
        TZ_CUDA(cudaMemsetAsync(p, 0, bytes ? bytes : 16, stream));      // padding columns stay finite
        return p;
    };
    r.row_inv = (float*)get(m * 4);
    r.x = (float*)get(m * h * 4);
    r.in = get(m * max_in * max_seg * es);
    r.proj = (float*)get(m * max_proj * 4);
    r.mix_a = get(m * max_mix * es);
    r.mix_b = get(m * max_mix * es);
    r.act = get(m * max_ff * es);
    r.ya = (float*)get(m * h * 4);
    r.yb = (float*)get(m * h * 4);
    r.cap = cap;
}

// ---- state ------------------------------------------------------------------------------------------------------------------
// A slot starts over by zeroing what its recurrences and convolutions carry; ring entries are only read below the position.
void HybridEngine::reset_seq(int s) {
    TZ_CUDA(cudaMemsetAsync(tails + (size_t)s * tail_floats, 0, tail_floats * 4, stream));
    TZ_CUDA(cudaMemsetAsync(states + (size_t)s * state_floats, 0, state_floats * 4, stream));
    seq_len[s] = 0;
}

void HybridEngine::reset_kv() {
    for (int s = 0; s < batch; ++s) reset_seq(s);
}

void HybridEngine::set_seq_len(int s, int len) {
    if (len == seq_len[s]) return;
    if (len != 0) throw std::invalid_argument("a recurrent state cannot be cut back or extended: reset the sequence and feed its tokens");
    reset_seq(s);
}

// ---- one walk through the layers ---------------------------------------------------------------------------------------------
RowsArgs HybridEngine::row_args(Pass& p, float gain, const float* conv, size_t tail) {
    RowsArgs a;
    a.width = h; a.M = p.M; a.eps = eps; a.gain = gain;
    a.conv_w = conv; a.taps = conv ? taps : 1;
    float* carried = tails + (size_t)p.seq * tail_floats + tail;
    a.tail_in = carried;
    a.tail_out = p.decode ? carried : tail_stage + tail;
    a.seq_stride = tail_floats;
    a.decode = p.decode;
    a.out = p.rows->in; a.ld_out = max_in;
    a.f32 = f32; a.use_pdl = p.decode && use_pdl;
    return a;
}

void HybridEngine::run_rows(Pass& p, RowsArgs& a) {
    if (p.embed) {
        a.tokens = p.tokens; a.pos = p.pos;
        a.embed = embed; a.pos_table = pos_table;
        a.vocab = V; a.n_pos = n_pos;
        p.embed = false;
    } else {
        a.x_in = p.rows->x;
        a.y0 = p.add.y0; a.y1 = p.add.y1; a.w0 = p.add.w0; a.w1 = p.add.w1;
        a.ld_y = h;
    }
    p.add = Pending();
    a.x_out = p.rows->x;
    a.row_inv = p.rows->row_inv;
    TZ_KERNEL(launch_rows(a, stream, &launches));
}

void HybridEngine::run_gemm(Pass& p, const void* a, const DenseWeight& w, void* c, int ld_c, const HybridLayer* mixes, const HybridLayer* act) {
    GemmArgs g;
    g.a = a; g.w = w.w; g.M = p.M; g.N = w.rows; g.ld_k = w.ld_k;
    g.seg_end[0] = w.rows;
    if (mixes) {
        g.n_seg = mixes->n_seg;
        std::copy(mixes->seg_end, mixes->seg_end + 8, g.seg_end);
        g.a_seg_stride = (size_t)p.M * w.ld_k;
    }
    if (act) { g.epilogue = TENZO_GEMM_XIELU; g.act_pos = act->act_pos; g.act_neg = act->act_neg; }
    g.c = c; g.ld_c = ld_c;
    g.f32 = f32; g.use_pdl = p.decode && use_pdl;
    g.workspace = gemm_ws; g.workspace_bytes = tenzo_cuda_gemm_workspace_bytes();
    TZ_KERNEL(launch_gemm(g, stream));
    launches += p.M > 8 && p.M < kGemmUmmaMinRows && !f32 ? 2 : 1;
}

void HybridEngine::run_layer(Pass& p, int l) {
    HybridLayer& y = layers[l];
    Rows& r = *p.rows;
    RowsArgs ra = row_args(p, y.norm1, y.canon1, y.tail1);
    if (y.n_mix) {
        ra.mu = y.mu; ra.n_mix = y.n_mix;
        float* carried = tails + (size_t)p.seq * tail_floats + y.prev;
        ra.prev_in = carried;
        ra.prev_out = p.decode ? carried : tail_stage + y.prev;
    }
    run_rows(p, ra);
    run_gemm(p, r.in, y.in, r.proj, max_proj, y.n_mix ? &y : nullptr);

    if (y.has_window) {
        const WindowMixer& m = y.win;
        WindowAttnArgs a;
        a.q = r.proj + m.off_q; a.k = r.proj + m.off_k; a.v = r.proj + m.off_v; a.ld = max_proj;
        a.conv_q = m.conv_q; a.conv_k = m.conv_k; a.conv_v = m.conv_v; a.taps = m.taps;
        float* carried = tails + (size_t)p.seq * tail_floats + m.tail;
        a.tail_in = carried;
        a.tail_out = p.decode ? carried : tail_stage + m.tail;
        a.tail_seq_stride = tail_floats;
        a.heads = m.heads; a.kv_heads = m.kv_heads; a.dim = m.dim; a.vdim = m.vdim; a.scale = m.scale;
        a.window = m.window; a.ring = m.ring;
        const size_t es = f32 ? 4 : 2;
        a.ring_k = static_cast<char*>(m.ring_k) + (size_t)p.seq * m.ring_k_stride * es;
        a.ring_v = static_cast<char*>(m.ring_v) + (size_t)p.seq * m.ring_v_stride * es;
        a.ring_k_stride = m.ring_k_stride; a.ring_v_stride = m.ring_v_stride;
        a.pos = p.pos; a.pos0 = p.pos0; a.M = p.M; a.decode = p.decode;
        a.out = r.mix_a; a.ld_out = m.o.ld_k;
        a.lin_q = lin_q; a.lin_k = lin_k; a.lin_v = lin_v;
        a.f32 = f32; a.use_pdl = p.decode && use_pdl;
        TZ_KERNEL(launch_window_attention(a, stream, &launches));
    }
    void* scan_out = y.has_window ? r.mix_b : r.mix_a;
    if (y.has_scan) {
        const ScanMixer& m = y.scan;
        ScanArgs a;
        a.q = r.proj + m.off_q; a.k = r.proj + m.off_k; a.v = r.proj + m.off_v; a.g = r.proj + m.off_g; a.ld = max_proj;
        a.q_scale = m.q_scale; a.k_scale = m.k_scale;
        a.heads = m.heads; a.dim = m.dim; a.vdim = m.vdim;
        a.decay_kind = m.decay_kind; a.decay = m.decay;
        a.low = r.proj + m.off_low; a.up = m.up; a.bias = m.bias; a.rank = m.rank; a.tau = m.tau;
        a.bonus = m.bonus; a.norm = m.norm; a.norm_per_head = m.norm_per_head; a.eps = eps;
        a.state = states + (size_t)p.seq * state_floats + m.state;
        a.state_seq_stride = state_floats;
        a.M = p.M; a.decode = p.decode;
        a.out = scan_out; a.ld_out = m.o.ld_k;
        a.w_rows = w_rows; a.o_rows = o_rows; a.part = scan_part;
        a.f32 = f32; a.use_pdl = p.decode && use_pdl;
        TZ_KERNEL(launch_scan(a, stream, &launches));
    }
    if (y.has_window && y.has_scan) {
        run_gemm(p, r.mix_a, y.win.o, r.ya, h);
        run_gemm(p, r.mix_b, y.scan.o, r.yb, h);
        p.add.y0 = r.ya; p.add.y1 = r.yb; p.add.w0 = y.left_out; p.add.w1 = y.right_out;
    } else {
        run_gemm(p, r.mix_a, y.has_window ? y.win.o : y.scan.o, r.ya, h);
        p.add.y0 = r.ya;
    }
    if (y.has_mlp) {
        RowsArgs rb = row_args(p, y.norm2, y.canon2, y.tail2);
        run_rows(p, rb);
        run_gemm(p, r.in, y.up, r.act, y.down.ld_k, nullptr, &y);
        run_gemm(p, r.act, y.down, r.ya, h);
        p.add.y0 = r.ya;
    }
}

void HybridEngine::enqueue_step(bool with_logits, bool feed_back, int) {
    Pass p = {&dec, batch, 1, 0, 0, d_tokens, d_pos};
    for (int l = 0; l < L; ++l) run_layer(p, l);
    RowsArgs ra = row_args(p, final_gain, nullptr, 0);
    run_rows(p, ra);
    if (with_logits) {
        run_gemm(p, dec.in, head, b_logits, V);
        TZ_KERNEL(launch_argmax(b_logits, V, batch, d_next, argmax_ws, stream));
        launches += 2;
    }
    enqueue_advance(feed_back);
}

void HybridEngine::enqueue_layer(int l, int) {
    Pass p = {&dec, batch, 1, 0, 0, d_tokens, d_pos};
    p.embed = false;
    run_layer(p, l);
    RowsArgs ra = row_args(p, 1.0f, nullptr, 0);
    run_rows(p, ra);
}

void HybridEngine::chunk_rows(int seq, const int* tokens, int M) {
    if (M > chunk.cap) {
        int cap = 64;
        while (cap < M) cap *= 2;
        alloc_rows(chunk, cap);
        chunk.cap = 0;                                 // until every buffer below exists too
        const size_t m = cap, es = f32 ? 4 : 2;
        auto get = [&](size_t bytes) -> void* {
            void* p = nullptr;
            TZ_CUDA(cudaMalloc(&p, bytes ? bytes : 16));
            chunk.owned.push_back(p);
            return p;
        };
        size_t lq = 0, lk = 0, lv = 0, w = 0, o = 0, part = 0;
        for (const HybridLayer& y : layers) {
            if (y.has_window) {
                const WindowMixer& a = y.win;
                lq = std::max(lq, m * a.heads * round_up(a.dim, 8));
                lk = std::max(lk, (m + a.ring) * a.kv_heads * round_up(a.dim, 8));
                lv = std::max(lv, (m + a.ring) * a.kv_heads * round_up(a.vdim, 8));
            }
            if (y.has_scan) {
                const ScanMixer& s = y.scan;
                if (s.decay_kind != TENZO_DECAY_CONST) w = std::max(w, m * s.heads * s.dim);
                o = std::max(o, m * s.heads * s.vdim);
                part = std::max(part, tenzo_cuda_linear_scan_part_floats(cap, s.heads, s.dim, s.vdim));
            }
        }
        chunk_tokens = (int*)get(m * 4);
        chunk_pos = (int*)get(m * 4);
        lin_q = get(lq * es);
        lin_k = get(lk * es);
        lin_v = get(lv * es);
        w_rows = (float*)get(w * 4);
        o_rows = (float*)get(o * 4);
        scan_part = (float*)get(part * 4);
        chunk.cap = cap;
    }
    const int pos0 = seq_len[seq];
    std::vector<int> hp(M);
    for (int i = 0; i < M; ++i) hp[i] = pos0 + i;
    TZ_CUDA(cudaMemcpyAsync(chunk_tokens, tokens, (size_t)M * 4, cudaMemcpyHostToDevice, stream));
    TZ_CUDA(cudaMemcpyAsync(chunk_pos, hp.data(), (size_t)M * 4, cudaMemcpyHostToDevice, stream));
    Pass p = {&chunk, M, 0, seq, pos0, chunk_tokens, chunk_pos};
    for (int l = 0; l < L; ++l) run_layer(p, l);
    RowsArgs ra = row_args(p, final_gain, nullptr, 0);
    run_rows(p, ra);                                   // leaves the normalised rows for rows_logits in chunk.in
    TZ_CUDA(cudaMemcpyAsync(tails + (size_t)seq * tail_floats, tail_stage, tail_floats * 4, cudaMemcpyDeviceToDevice, stream));
    TZ_CUDA(cudaMemcpyAsync(dec.x + (size_t)seq * h, chunk.x + (size_t)(M - 1) * h, (size_t)h * 4, cudaMemcpyDeviceToDevice, stream));
    TZ_CUDA(cudaStreamSynchronize(stream));
    if (tenzo_cuda_gemm_take_timeouts() > 0) throw std::runtime_error("a matrix product gave up waiting for a tile copy; results are invalid");
    seq_len[seq] += M;
}

void HybridEngine::rows_logits(const int* want, int n_want, float* host) {
    const size_t row = (size_t)max_in * (f32 ? 4 : 2);
    constexpr int kGroup = 128;
    if (!logit_in) {
        logit_in = dalloc(kGroup * row);
        want_logits = (float*)dalloc((size_t)kGroup * V * 4);
    }
    for (int a = 0; a < n_want; a += kGroup) {
        const int n = std::min(kGroup, n_want - a);
        for (int i = 0; i < n;) {                      // runs of neighbouring rows
            int j = i + 1;
            while (j < n && want[a + j] == want[a + j - 1] + 1) ++j;
            TZ_CUDA(cudaMemcpyAsync(static_cast<char*>(logit_in) + i * row, static_cast<char*>(chunk.in) + (size_t)want[a + i] * row,
                                    (size_t)(j - i) * row, cudaMemcpyDeviceToDevice, stream));
            i = j;
        }
        Pass p = {&chunk, n, 0, 0, 0, nullptr, nullptr};
        run_gemm(p, logit_in, head, want_logits, V);
        TZ_CUDA(cudaMemcpyAsync(host + (size_t)a * V, want_logits, (size_t)n * V * 4, cudaMemcpyDeviceToHost, stream));
    }
    TZ_CUDA(cudaStreamSynchronize(stream));
}

const float* HybridEngine::buffer(int which, int seq, size_t* n) {
    switch (which) {
        case TENZO_BUF_X: *n = h; return dec.x + (size_t)seq * h;
        case TENZO_BUF_LOGITS: *n = V; return b_logits + (size_t)seq * V;
        default: throw std::invalid_argument("this model keeps no such buffer");
    }
}

void HybridEngine::check_device_status(bool force) {
    // only launches of 16 and more rows have bounded waits; single-sequence decode is polled now and then
    if (!force && batch == 1 && (++status_poll & 31) != 0) return;
    if (tenzo_cuda_gemm_take_timeouts() > 0) throw std::runtime_error("a matrix product gave up waiting for a tile copy; results are invalid");
}

static EngineCore* open_sozopel(const Json& config, const OpenOptions& o) { return new HybridEngine(config, o); }
static const ModelRegistration registration({"Sozopel", open_sozopel});

}  // namespace tz

// Hybrid decoders on the shared engine (hybrid_engine.h): weights, state and the walk through the layers.
//
// One layer, M rows (decode: one per sequence; chunk: consecutive tokens of one sequence):
//   rows     x += what the previous sublayer left (normed first, in some designs), norm1, convolution (, token-shift mixes)
//   gemm     every projection of the mixer's input in one product
//   window   convolution on q, k, v, ring update, attention          }
//   latent   latent cache row, attention over latents or expanded     } whichever the mixer has
//   scan     decays, recurrence, per-head norm, gate                  }
//   delta    convolutions, delta rule, per-head norm, gate            }
//   gemm     output projection(s)
//   rows, gemm (+ activation), gemm    the feed-forward, when the layer has one; a mixture of experts: rows, gemm (router),
//                                      route, two grouped gemms
// Residual sums happen at the start of the next row kernel.
#include "hybrid_engine.h"

#include <algorithm>
#include <cmath>
#include <cstring>

namespace tz {

HybridEngine::HybridEngine(const Json& config, const OpenOptions& o, Loader load) {
    try {
        init(config, o, load);
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

void HybridEngine::init(const Json& c, const OpenOptions& o, Loader load) {
    f32 = o.compute == TENZO_COMPUTE_F32;
    init_core(o.opt.batch, o.opt.use_graph, o.opt.use_pdl);
    (this->*load)(c, SafeTensors(o.dir + "/model.safetensors"));
    cfg = {};
    cfg.hidden_size = h;
    cfg.vocab_size = V;
    cfg.num_layers = L;
    cfg.max_seq_len = n_pos;
    cfg.kv_mode = f32 ? "window_f32" : "window_bf16";
    cfg.device = "cuda";
    init_core_buffers();
    tail_floats = std::max<size_t>(tail_floats, 4);
    state_floats = std::max<size_t>(state_floats, 4);
    for (const HybridLayer& y : layers) {
        if (y.has_window) max_mix = std::max(max_mix, y.win.o.ld_k);
        if (y.has_scan) max_mix = std::max(max_mix, y.scan.o.ld_k);
        if (y.has_delta) max_mix = std::max(max_mix, y.delta.o.ld_k);
        if (y.has_latent) {
            max_mix = std::max(max_mix, y.lat.o.ld_k);
            max_lat = std::max(max_lat, (size_t)y.lat.heads * caches[y.lat.cache].ld_c());
        }
        if (y.moe.experts) {
            max_top = std::max(max_top, y.moe.top);
            max_experts = std::max(max_experts, y.moe.experts);
            max_expert_ff = std::max(max_expert_ff, y.moe.down.ld_k);
            max_proj = std::max(max_proj, round_up(y.moe.experts, 8));
        } else if (y.has_mlp) {
            max_ff = std::max(max_ff, y.down.ld_k);
        }
    }

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
    int n_lin = 1;                                     // chunk buffers: 0 is shared by the caches that nobody borrows
    for (LatentCache& k : caches) {
        k.ring_c_stride = (size_t)k.ring * k.ld_c();
        k.ring_r_stride = (size_t)k.ring * k.rot8();
        k.ring_c = dalloc(B * k.ring_c_stride * es);
        k.ring_r = dalloc(B * k.ring_r_stride * es);
        k.lin = k.borrowed ? n_lin++ : 0;
    }
    lin_c.assign(caches.empty() ? 0 : n_lin, nullptr);
    lin_r = lin_c;
    gemm_ws = dalloc(tenzo_cuda_gemm_workspace_bytes());
    argmax_ws = dalloc(argmax_scratch_bytes(batch));
    alloc_rows(dec, batch);
    if (max_lat) {
        dec.q_abs = (float*)dalloc(B * max_lat * 4);
        dec.lat = dalloc(B * max_lat * es);
    }
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

size_t HybridEngine::take_tail(size_t floats) {
    const size_t at = tail_floats;
    tail_floats += (floats + 3) / 4 * 4;
    return at;
}

size_t HybridEngine::take_state(size_t floats) {
    const size_t at = state_floats;
    state_floats += (floats + 3) / 4 * 4;
    return at;
}

void HybridEngine::start_layers(int n) {
    L = n;
    if (h <= 0 || V <= 0 || n_pos <= 0 || L <= 0) throw std::invalid_argument("non-positive dimension");
    layers.resize(L);
    max_in = round_up(h, 64);
}

// Every projection of a mixer's input as one product, pieces at multiples of `align` columns. With mixes each piece multiplies
// its own one: a segment of the product.
void HybridEngine::fuse_inputs(HybridLayer& y, const std::vector<Piece>& pieces, int align, const SafeTensors& st) {
    int n = 0;
    y.n_seg = 0;
    for (size_t i = 0; i < pieces.size(); ++i) {
        *pieces[i].off = n;
        n += i + 1 < pieces.size() ? round_up(pieces[i].rows, align) : pieces[i].rows;
        if (y.n_mix) y.seg_end[y.n_seg++] = n;
    }
    if (!y.n_mix) y.seg_end[y.n_seg++] = n;
    y.in = make_weight(n, h);
    for (const Piece& q : pieces) upload_weight(y.in, *q.off, st, q.name, q.rows, h);
    max_proj = std::max(max_proj, round_up(n, 8));
    max_seg = std::max(max_seg, std::max(1, y.n_mix));
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
    if (max_top) {
        const size_t pairs = m * max_top;
        r.chosen = (int*)get(pairs * 4);
        r.slot = (int*)get(pairs * 4);
        r.row_of = (int*)get(pairs * 4);
        r.group_off = (int*)get((max_experts + 1) * 4);
        r.weight = (float*)get(pairs * 4);
        r.ye = (float*)get(pairs * h * 4);
        r.act_e = get(pairs * max_expert_ff * es);
        if (!f32) r.gathered = get(pairs * max_in * es);
    }
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
RowsArgs HybridEngine::row_args(Pass& p, float gain, const float* gain_w, const float* conv, size_t tail) {
    RowsArgs a;
    a.width = h; a.M = p.M; a.eps = eps; a.gain = gain; a.gain_w = gain_w;
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
        a.y_slot = p.add.slot; a.y_weight = p.add.weight; a.n_y = p.add.n_y;
        a.ld_y = h;
    }
    p.add = Pending();
    a.x_out = p.rows->x;
    a.row_inv = p.rows->row_inv;
    TZ_KERNEL(launch_rows(a, stream, &launches));
}

GemmArgs HybridEngine::gemm_args(Pass& p, const void* a, const DenseWeight& w, void* c, int ld_c) {
    GemmArgs g;
    g.a = a; g.w = w.w; g.M = p.M; g.N = w.rows; g.ld_k = w.ld_k;
    g.seg_end[0] = w.rows;
    g.c = c; g.ld_c = ld_c;
    g.f32 = f32; g.use_pdl = p.decode && use_pdl;
    g.workspace = gemm_ws; g.workspace_bytes = tenzo_cuda_gemm_workspace_bytes();
    return g;
}

void HybridEngine::run_gemm(const GemmArgs& g) { TZ_KERNEL(launch_gemm(g, stream, &launches)); }

void HybridEngine::run_window(Pass& p, HybridLayer& y) {
    Rows& r = *p.rows;
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

void HybridEngine::run_scan(Pass& p, HybridLayer& y) {
    Rows& r = *p.rows;
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
    a.out = y.has_window ? r.mix_b : r.mix_a; a.ld_out = m.o.ld_k;
    a.w_rows = w_rows; a.o_rows = o_rows; a.part = scan_part;
    a.f32 = f32; a.use_pdl = p.decode && use_pdl;
    TZ_KERNEL(launch_scan(a, stream, &launches));
}

void HybridEngine::run_delta(Pass& p, HybridLayer& y) {
    Rows& r = *p.rows;
    const DeltaMixer& m = y.delta;
    DeltaArgs a;
    a.q = r.proj + m.off_q; a.k = r.proj + m.off_k; a.v = r.proj + m.off_v; a.g = r.proj + m.off_g; a.a = r.proj + m.off_a; a.b = r.proj + m.off_b;
    a.ld = max_proj;
    a.conv_q = m.conv_q; a.conv_k = m.conv_k; a.conv_v = m.conv_v; a.taps = m.taps;
    float* slot = states + (size_t)p.seq * state_floats;
    a.tail = slot + m.tail; a.tail_seq_stride = state_floats;
    a.heads = m.heads; a.kv_heads = m.kv_heads; a.dim = m.dim; a.vdim = m.vdim;
    a.q_scale = (float)std::pow((double)m.dim, -0.5);
    a.a_log = m.a_log; a.dt_bias = m.dt_bias; a.norm = m.norm; a.eps = eps;
    a.state = slot + m.state; a.state_seq_stride = state_floats;
    a.pos = p.pos; a.pos0 = p.pos0; a.M = p.M; a.decode = p.decode;
    a.out = r.mix_a; a.ld_out = m.o.ld_k;
    a.work = delta_work;
    a.f32 = f32; a.use_pdl = p.decode && use_pdl;
    TZ_KERNEL(launch_delta(a, stream, &launches));
}

void HybridEngine::run_latent(Pass& p, HybridLayer& y) {
    Rows& r = *p.rows;
    const LatentMixer& m = y.lat;
    const LatentCache& k = caches[m.cache];
    LatentAttnArgs a;
    a.q = r.proj + m.off_q; a.dkv = m.owner ? r.proj + m.off_dkv : nullptr; a.ld = max_proj;
    a.norm = m.norm; a.eps = eps; a.freq = k.freq;
    a.heads = m.heads; a.dim = m.dim; a.rot = k.rot; a.vdim = m.vdim; a.rank = k.rank;
    a.scale = m.scale; a.window = m.window; a.w_kv = m.kv;
    const size_t es = f32 ? 4 : 2;
    a.ring_c = static_cast<char*>(k.ring_c) + (size_t)p.seq * k.ring_c_stride * es;
    a.ring_r = static_cast<char*>(k.ring_r) + (size_t)p.seq * k.ring_r_stride * es;
    a.ring = k.ring; a.ring_c_stride = k.ring_c_stride; a.ring_r_stride = k.ring_r_stride;
    a.pos = p.pos; a.pos0 = p.pos0; a.M = p.M; a.decode = p.decode;
    a.out = r.mix_a; a.ld_out = m.o.ld_k;
    a.lin_q = lin_q; a.lin_c = lin_c[k.lin]; a.lin_r = lin_r[k.lin]; a.kv = lat_kv;
    a.q_abs = r.q_abs; a.lat = r.lat;
    a.workspace = gemm_ws; a.workspace_bytes = tenzo_cuda_gemm_workspace_bytes();
    a.f32 = f32; a.use_pdl = p.decode && use_pdl;
    TZ_KERNEL(launch_latent_attention(a, stream, &launches));
}

// The chosen experts of every row; their outputs are weighted and summed by the next row kernel.
void HybridEngine::run_experts(Pass& p, HybridLayer& y) {
    Rows& r = *p.rows;
    const ExpertMlp& m = y.moe;
    run_gemm(gemm_args(p, r.in, m.router, r.proj, max_proj));
    RouteArgs a;
    a.logits = r.proj; a.ld = max_proj; a.correction = m.correction;
    a.experts = m.experts; a.top = m.top; a.M = p.M;
    a.chosen = r.chosen; a.weight = r.weight; a.slot = r.slot; a.row_of = r.row_of; a.group_off = r.group_off;
    a.use_pdl = p.decode && use_pdl;
    TZ_KERNEL(launch_route(a, stream, &launches));
    GemmArgs g = gemm_args(p, r.in, m.up, r.act_e, m.down.ld_k);
    g.M = p.M * m.top; g.N = 2 * m.ff; g.seg_end[0] = g.N;
    g.epilogue = TENZO_GEMM_GLU_SILU;
    g.group_off = r.group_off; g.n_group = m.experts;
    g.a_index = r.row_of; g.a_rows = p.M; g.a_gather = r.gathered;
    run_gemm(g);
    g = gemm_args(p, r.act_e, m.down, r.ye, h);
    g.M = p.M * m.top; g.N = h; g.seg_end[0] = g.N;
    g.group_off = r.group_off; g.n_group = m.experts;
    run_gemm(g);
    p.add.y0 = r.ye; p.add.slot = r.slot; p.add.weight = r.weight; p.add.n_y = m.top;
}

void HybridEngine::run_layer(Pass& p, int l) {
    HybridLayer& y = layers[l];
    Rows& r = *p.rows;
    RowsArgs ra = row_args(p, y.norm1, y.norm1_w, y.canon1, y.tail1);
    if (y.n_mix) {
        ra.mu = y.mu; ra.n_mix = y.n_mix;
        float* carried = tails + (size_t)p.seq * tail_floats + y.prev;
        ra.prev_in = carried;
        ra.prev_out = p.decode ? carried : tail_stage + y.prev;
    }
    run_rows(p, ra);
    GemmArgs in = gemm_args(p, r.in, y.in, r.proj, max_proj);
    if (y.n_mix) {
        in.n_seg = y.n_seg;
        std::copy(y.seg_end, y.seg_end + 8, in.seg_end);
        in.a_seg_stride = (size_t)p.M * y.in.ld_k;
    }
    run_gemm(in);
    if (y.has_window) run_window(p, y);
    if (y.has_scan) run_scan(p, y);
    if (y.has_delta) run_delta(p, y);
    if (y.has_latent) run_latent(p, y);
    if (y.has_window && y.has_scan) {
        run_gemm(gemm_args(p, r.mix_a, y.win.o, r.ya, h));
        run_gemm(gemm_args(p, r.mix_b, y.scan.o, r.yb, h));
        p.add.y0 = r.ya; p.add.y1 = r.yb; p.add.w0 = y.left_out; p.add.w1 = y.right_out;
    } else {
        run_gemm(gemm_args(p, r.mix_a, y.has_window ? y.win.o : y.has_scan ? y.scan.o : y.has_delta ? y.delta.o : y.lat.o, r.ya, h));
        p.add.y0 = r.ya; p.add.w0 = y.post1_w;
    }
    if (!y.has_mlp) return;
    RowsArgs rb = row_args(p, y.norm2, y.norm2_w, y.canon2, y.tail2);
    run_rows(p, rb);
    if (y.moe.experts) {
        run_experts(p, y);
    } else {
        GemmArgs up = gemm_args(p, r.in, y.up, r.act, y.down.ld_k);
        up.epilogue = y.up_epilogue; up.act_pos = y.act_pos; up.act_neg = y.act_neg;
        run_gemm(up);
        run_gemm(gemm_args(p, r.act, y.down, r.ya, h));
        p.add.y0 = r.ya;
    }
    p.add.w0 = y.post2_w;
}

// Leaves the normalised rows in p.rows->in.
void HybridEngine::run_final(Pass& p) {
    RowsArgs ra = row_args(p, final_gain, final_gain_w, nullptr, 0);
    run_rows(p, ra);
}

void HybridEngine::run_head(Pass& p, const void* rows, float* logits) {
    GemmArgs g = gemm_args(p, rows, head, logits, V);
    if (logit_cap > 0.0f) { g.epilogue = TENZO_GEMM_SOFTCAP; g.cap = logit_cap; }
    run_gemm(g);
}

void HybridEngine::enqueue_step(bool with_logits, bool feed_back, int) {
    Pass p = {&dec, batch, 1, 0, 0, d_tokens, d_pos};
    for (int l = 0; l < L; ++l) run_layer(p, l);
    run_final(p);
    if (with_logits) {
        run_head(p, dec.in, b_logits);
        TZ_KERNEL(launch_argmax(b_logits, V, batch, d_next, argmax_ws, stream));
        launches += 2;
    }
    enqueue_advance(feed_back);
}

void HybridEngine::enqueue_layer(int l, int) {
    Pass p = {&dec, batch, 1, 0, 0, d_tokens, d_pos};
    p.embed = false;
    run_layer(p, l);
    RowsArgs ra = row_args(p, 1.0f, nullptr, nullptr, 0);
    run_rows(p, ra);
}

// Activations and scratch of chunks of up to `rows` rows.
void HybridEngine::grow_chunk(int rows) {
    if (rows <= chunk.cap) return;
    int cap = 64;
    while (cap < rows) cap *= 2;
    alloc_rows(chunk, cap);
    chunk.cap = 0;                                     // until every buffer below exists too
    const size_t m = cap, es = f32 ? 4 : 2;
    auto get = [&](size_t bytes) -> void* {
        void* p = nullptr;
        TZ_CUDA(cudaMalloc(&p, bytes ? bytes : 16));
        chunk.owned.push_back(p);
        return p;
    };
    size_t lq = 0, lk = 0, lv = 0, w = 0, o = 0, part = 0, work = 0, kv = 0;
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
        if (y.has_delta) work = std::max(work, tenzo_cuda_delta_rule_work_floats(cap, y.delta.heads, y.delta.kv_heads, y.delta.dim, y.delta.vdim));
        if (y.has_latent) {
            const LatentMixer& a = y.lat;
            lq = std::max(lq, m * a.heads * (a.dim8() + caches[a.cache].rot8()));
            kv = std::max(kv, (m + std::min(a.window, n_pos)) * a.heads * (a.dim8() + a.vdim8()));
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
    delta_work = (float*)get(work * 4);
    lat_kv = get(kv * es);
    for (size_t i = 0; i < lin_c.size(); ++i) {
        size_t c = 0, r = 0;
        for (const LatentCache& k : caches)
            if (k.lin == (int)i) {
                c = std::max(c, (m + k.ring) * k.ld_c());
                r = std::max(r, (m + k.ring) * k.rot8());
            }
        lin_c[i] = get(c * es);
        lin_r[i] = get(r * es);
    }
    chunk.cap = cap;
}

void HybridEngine::chunk_rows(int seq, const int* tokens, int M) {
    grow_chunk(M);
    const int pos0 = seq_len[seq];
    std::vector<int> hp(M);
    for (int i = 0; i < M; ++i) hp[i] = pos0 + i;
    TZ_CUDA(cudaMemcpyAsync(chunk_tokens, tokens, (size_t)M * 4, cudaMemcpyHostToDevice, stream));
    TZ_CUDA(cudaMemcpyAsync(chunk_pos, hp.data(), (size_t)M * 4, cudaMemcpyHostToDevice, stream));
    Pass p = {&chunk, M, 0, seq, pos0, chunk_tokens, chunk_pos};
    for (int l = 0; l < L; ++l) run_layer(p, l);
    run_final(p);                                      // for rows_logits
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
        run_head(p, logit_in, want_logits);
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

}  // namespace tz

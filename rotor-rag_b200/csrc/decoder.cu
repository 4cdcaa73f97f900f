// Driver of layer-described decoders: a list of layer runs (a layer may run several times in a row with
// the same weights, each run with its own cache), residual streams with hyper-connections or one residual
// whose two sublayers read the same row, bias or latent attention, a gated feed-forward or routed experts,
// an output head.  It sits behind the same model handle as the ternary model: position state, generation
// loop, token log and captured graph are handle.cu's.
//
// Launch sequence of a forward, per layer run
//   many rows:  stage (streams, norms) -> input product -> mixer -> o product -> feed-forward (with a stage in
//               front where the sublayers follow one another)
//   up to DENSE_FEW_ROWS rows: the stages ride in the input products' prologues
// Mixers, many rows / generation step
//   bias:    [head finish ->] attention              / attention (normalises and appends its own row)
//   latent:  [query latent norm, product (rotates) ->] finish -> expansion of the cached latents -> attention (prompts), or
//            finish -> absorbing product -> attention -> value product
//                                                    / [product ->] absorbing product -> attention (rotates,
//                                                      norms and appends its own row) -> value product
// Feed-forwards
//   dense:   gate/up product (gating in its read-back) -> down product
//   experts: router product -> choice, table, scatter -> the same two products over the experts' slots (the stage
//            that follows adds a token's slots up)    / router rows in the input product -> gate/up product of
//            each token's choices -> their weighted down product
// then a stage that sums the streams and applies the final norm on the rows whose logits are wanted, and
// the LM head.  Streams alternate between two buffers.
#include <cstdlib>
#include <cstring>
#include <new>
#include <vector>

#include "decoder.cuh"
#include "model_handle.cuh"

namespace rb {

struct DecoderStack {
    rotor_b200_decoder_config cfg;
    std::vector<rotor_b200_decoder_layer> layers;
    std::vector<rotor_b200_decoder_run> runs;
    const __nv_bfloat16* embed;  // [vocab][ld]
    const __nv_bfloat16* head;   // [vocab][ldh]
    const float* final_norm;     // [ld]
    int ld, ldh;                 // width rounded to DENSE_LD; to the LM head's 256 columns
    // workspace
    float* x[2];                 // residual streams [rows][streams][ld]
    float *y, *y2;               // sublayer outputs [rows][ld]
    void *h, *h2;                // sublayer inputs [rows][ld]
    float* qkv;                  // raw projections
    __nv_bfloat16* q;            // normalised queries
    void* attn;                  // attention rows
    void* act;                   // gated rows
    float* gate_up;              // float32 runs: both halves before the gating
    // latent attention
    float* q_raw;                // queries made from their latents
    void *cq, *lq;               // normed query latents; rotated query rows
    void *q_abs, *o_lat;         // absorbed queries, weighted latents (abs_rows of them)
    __nv_bfloat16* kv;           // expanded keys and values [kv_rows]
    int abs_rows, kv_rows;
    bool absorb_all;             // workspace for prompts in the absorbed form too
    // experts
    float* logits;               // router outputs [rows][lde]
    void *perm, *slots;          // rows by slot; their outputs
    Routing route;
    float* hn;                   // final rows [rows][ldh]
    int* row_map;
    std::vector<int> host_map;
};

static HeadShape shape_of(const rotor_b200_decoder_layer& L, float eps) {
    HeadShape s;
    s.heads = L.heads;
    s.kv_heads = L.kv_heads;
    s.dim = L.dim;
    s.vdim = L.vdim;
    s.kd = (L.dim + 7) / 8 * 8;
    s.vd = (L.vdim + 7) / 8 * 8;
    s.unit = L.unit_qk;
    s.eps = eps;
    return s;
}

static int up(int n, int to) { return (n + to - 1) / to * to; }

static LatentShape latent_of(const rotor_b200_decoder_layer& L, float eps) {
    LatentShape s;
    s.heads = L.heads;
    s.dim = L.dim;
    s.rot = L.rot_dim;
    s.vdim = L.vdim;
    s.rank = L.kv_rank;
    s.dp = up(L.dim, 8);
    s.rp = up(L.rot_dim, 16);
    s.kp = up(L.kv_rank, 16);
    s.eps = eps;
    return s;
}

static bool is_latent(const rotor_b200_decoder_layer& L) { return L.mixer == ROTOR_B200_MIXER_LATENT; }

// Columns of a latent layer's input product: queries (or their latents), cache row, gates.
struct LatentColumns {
    int q, dkv, all;
};
static LatentColumns latent_columns(const rotor_b200_decoder_layer& L) {
    const LatentShape s = latent_of(L, 0.f);
    LatentColumns c;
    c.q = L.q_rank ? up(L.q_rank, 16) : s.heads * latent_q(s);
    c.dkv = L.own_kv ? latent_row(s) : 0;
    c.all = c.q + c.dkv + (L.gated ? s.heads : 0);
    return c;
}
// Columns of a mixer's output row.
static int mixer_cols(const rotor_b200_decoder_layer& L) { return L.heads * (is_latent(L) ? up(L.vdim, 8) : L.vdim); }

static int check_decoder(const rotor_b200_decoder_config& c, const rotor_b200_decoder_layer* layers,
                         const rotor_b200_decoder_run* runs) {
    if (c.vocab_size <= 0 || c.width <= 0 || c.streams < 1 || c.streams > STREAMS_MAX || c.n_layers <= 0 || c.n_runs <= 0 ||
        c.max_batch <= 0 || c.max_seq <= 0 || c.max_rows <= 0)
        return ROTOR_B200_ERR_ARG;
    if (c.width > 10240) return ROTOR_B200_ERR_SHAPE;  // a row of the stage kernel lives in shared memory
    for (int l = 0; l < c.n_layers; ++l) {
        const rotor_b200_decoder_layer& L = layers[l];
        if (L.heads <= 0 || L.kv_heads <= 0 || L.heads % L.kv_heads || L.dim <= 0 || L.vdim <= 0 || L.ff < 0 || L.chunk < 0)
            return ROTOR_B200_ERR_ARG;
        if (L.dim > 512 || L.vdim > 512) return ROTOR_B200_ERR_SHAPE;
        if (L.window < 0 || (L.parallel && c.streams != 1) || (L.ff && (L.norm1_b != nullptr) != (L.norm2_b != nullptr)) ||
            (L.act != ROTOR_B200_ACT_GELU_TANH && L.act != ROTOR_B200_ACT_SILU))
            return ROTOR_B200_ERR_ARG;
        if (L.experts && (!L.ff || L.experts < 0 || L.top < 1 || L.top > L.experts)) return ROTOR_B200_ERR_ARG;
        if (L.experts > EXPERTS_MAX || (L.experts && L.top > EXPERT_TOP_MAX)) return ROTOR_B200_ERR_SHAPE;
        if (is_latent(L)) {
            if (L.kv_rank <= 0 || L.rot_dim < 0 || L.rot_dim % 2 || L.q_rank < 0) return ROTOR_B200_ERR_ARG;
            if (!latent_attn_supported(latent_of(L, c.eps), c.f32)) return ROTOR_B200_ERR_SHAPE;
        } else if (L.mixer != ROTOR_B200_MIXER_BIAS) {
            return ROTOR_B200_ERR_ARG;
        }
    }
    if (runs)
        for (int r = 0; r < c.n_runs; ++r)
            if (runs[r].layer < 0 || runs[r].layer >= c.n_layers || !runs[r].k_cache || (!runs[r].v_cache && !is_latent(layers[runs[r].layer])))
                return ROTOR_B200_ERR_ARG;
    return ROTOR_B200_OK;
}

static void carve_decoder(Model& m, DecoderStack& d, const rotor_b200_decoder_layer* layers, unsigned char* base, size_t* total) {
    const rotor_b200_decoder_config& c = d.cfg;
    const size_t rows = c.max_rows, esz = c.f32 ? 4 : 2;
    struct {  // widest of every kind of row, in elements
        size_t qkv = 0, q = 0, attn = 0, act = 0, gu = 0, q_raw = 0, cq = 0, lq = 0, abs = 0, lat = 0, kv = 0, lde = 0, slots = 0, experts = 0, top = 0;
    } w;
    auto widen = [](size_t& v, size_t n) { v = n > v ? n : v; };
    bool parallel = false, absorb_all = d.absorb_all;
    for (int l = 0; l < c.n_layers; ++l) {
        const rotor_b200_decoder_layer& L = layers[l];
        parallel |= L.parallel != 0;
        if (is_latent(L)) {
            const LatentShape s = latent_of(L, c.eps);
            widen(w.qkv, dense_ld(latent_columns(L).all));
            if (L.q_rank) {
                widen(w.q_raw, dense_ld(s.heads * latent_q(s)));
                widen(w.cq, dense_ld(L.q_rank));
            }
            widen(w.lq, (size_t)s.heads * latent_q(s));
            widen(w.abs, (size_t)s.heads * latent_row(s));
            widen(w.lat, (size_t)s.heads * s.kp);
            if (!c.f32 && expanded_attn_supported(s, 16))
                widen(w.kv, (size_t)s.heads * (s.dp + up(s.vdim, 8)));
            else
                absorb_all = true;
        } else {
            const HeadShape s = shape_of(L, c.eps);
            widen(w.qkv, dense_ld(head_cols(s)));
            if (!c.f32) widen(w.q, (size_t)s.heads * s.kd);
        }
        widen(w.attn, dense_ld(mixer_cols(L)));
        const size_t per = L.experts ? L.top : 1;
        widen(w.act, per * dense_ld(L.ff));
        widen(w.gu, per * 2 * L.ff);
        if (L.experts) {
            widen(w.lde, dense_ld(L.experts));
            widen(w.slots, per * dense_ld(c.width));
            widen(w.experts, L.experts);
            widen(w.top, per);
        }
    }
    d.ld = dense_ld(c.width);
    d.ldh = (c.width + 255) / 256 * 256;
    Carve cv{base, 0};
    auto bytes = [&](size_t n) -> void* { return n ? cv.take<unsigned char>(n) : nullptr; };
    for (int i = 0; i < 2; ++i) d.x[i] = cv.take<float>(rows * c.streams * d.ld);
    d.y = cv.take<float>(rows * d.ld);
    d.y2 = static_cast<float*>(bytes(parallel ? rows * d.ld * 4 : 0));
    d.h = bytes(rows * d.ld * esz);
    d.h2 = bytes(parallel ? rows * d.ld * esz : 0);
    d.qkv = cv.take<float>(rows * w.qkv);
    d.q = static_cast<__nv_bfloat16*>(bytes(rows * w.q * 2));
    d.attn = bytes(rows * w.attn * esz);
    d.act = bytes(rows * w.act * esz);
    d.gate_up = static_cast<float*>(bytes(c.f32 ? rows * w.gu * 4 : 0));
    d.q_raw = static_cast<float*>(bytes(rows * w.q_raw * 4));
    d.cq = bytes(rows * w.cq * esz);
    d.lq = bytes(rows * w.lq * esz);
    const size_t short_rows = (size_t)c.max_batch * 15;  // (longer portions are expanded)
    d.abs_rows = (int)(absorb_all || short_rows > rows ? rows : short_rows);
    d.q_abs = bytes(d.abs_rows * w.abs * esz);
    d.o_lat = bytes(d.abs_rows * w.lat * esz);
    const size_t most = (size_t)c.max_batch * c.max_seq, some = rows > (size_t)c.max_seq ? rows : (size_t)c.max_seq;
    d.kv_rows = (int)(most < some ? most : some);
    d.kv = static_cast<__nv_bfloat16*>(bytes(d.kv_rows * w.kv * 2));
    d.logits = static_cast<float*>(bytes(rows * w.lde * 4));
    d.perm = bytes(rows * w.slots * esz);
    d.slots = bytes(rows * w.slots * esz);
    memset(&d.route, 0, sizeof(d.route));
    if (w.experts) {
        d.route.slot_of = cv.take<int>(rows * w.top);
        d.route.weight = cv.take<float>(rows * w.top);
        d.route.chosen = cv.take<int>(rows * w.top);
        d.route.counts = cv.take<int>(w.experts);
        d.route.cursor = cv.take<int>(w.experts);
        d.route.tile_rows = c.f32 ? 64 : 128;
        d.route.max_tiles = route_tiles((long long)(rows * w.top), (int)w.experts, d.route.tile_rows);
        d.route.table = cv.take<int>(1 + 3 * (size_t)d.route.max_tiles);
    }
    d.hn = cv.take<float>(rows * d.ldh);
    d.row_map = cv.take<int>(rows);
    const size_t nparts = (size_t)(lmhead_parts() > lmhead_mma_parts(c.vocab_size) ? lmhead_parts() : lmhead_mma_parts(c.vocab_size));
    m.part_val = cv.take<float>(rows * nparts);
    m.part_idx = cv.take<int>(rows * nparts);
    // (float32 runs keep the few-row LM head, which multiplies in float32)
    m.xsplit = rows > 4 && !c.f32 ? cv.take<__nv_bfloat16>(2 * rows * (size_t)d.ldh) : nullptr;
    m.c.d_pos = cv.take<int>(c.max_batch);
    m.c.counters = cv.take<unsigned>(8 + (size_t)c.max_batch);
    m.cur_ids = cv.take<long long>(c.max_batch);
    m.max_log = c.max_seq;
    m.tok_log = cv.take<long long>((size_t)m.max_log * c.max_batch);
    m.d_step = cv.take<int>(1);
    m.d_lens = cv.take<int>(c.max_batch);
    *total = cv.off;
}

// One forward on its way through the layers.
struct DecoderPass {
    Model& m;
    DecoderStack& d;
    int batch, seq, rows, f32;
    bool few;
    cudaStream_t st;
    StreamStage sg;
    int cur = 0;           // stream buffer the next stage writes
    bool routed = false;   // the router's outputs of the layer at hand are there
    int expand = -1;       // latent attention: 0 absorbed, 1 expanded, -1 by what is at hand

    DecoderPass(Model& m_, DecoderStack& d_, int batch_, int seq_, cudaStream_t st_)
        : m(m_), d(d_), batch(batch_), seq(seq_), rows(batch_ * seq_), f32(d_.cfg.f32), few(rows <= DENSE_FEW_ROWS && !m_.no_fused), st(st_), sg() {
        const rotor_b200_decoder_config& c = d.cfg;
        sg.streams = c.streams;
        sg.n = c.width;
        sg.ld = d.ld;
        sg.embed = d.embed;
        sg.vocab = c.vocab_size;
        sg.embed_scale = c.embed_scale;
        sg.eps = c.eps;
        sg.y = d.y;
        sg.h = d.h;
        sg.ldh = d.ld;
        sg.h_f32 = f32;
    }

    // points the stage at the sublayer that follows; the caller runs it
    void stage(const float* in, const float* norm, const float* norm_b) {
        sg.in = in;
        sg.norm = norm;
        sg.norm_b = norm_b;
        sg.norm2 = sg.norm2_b = nullptr;
        sg.x_in = d.x[cur ^ 1];
        sg.x_out = d.x[cur];
    }
    // after the stage has run: the coefficients of the sublayer whose output the next stage adds
    void after(const float* mix, const float* out) {
        sg.ids = nullptr;
        sg.mix = mix;
        sg.out = out;
        sg.y = d.y;
        sg.y2 = nullptr;
        sg.slots = nullptr;
        cur ^= 1;
    }

    DenseProduct product(const void* w, int n, int k, const void* x, int ldx) const {
        DenseProduct p = {};
        p.w = static_cast<const __nv_bfloat16*>(w);
        p.n = n;
        p.k = k;
        p.ldw = dense_ld(k);
        p.f32 = f32;
        p.x = x;
        p.ldx = ldx;
        return p;
    }
    DenseProduct plain(const void* w, int n, int k, const void* x, int ldx, float* y, int ldy) const {
        DenseProduct p = product(w, n, k, x, ldx);
        p.y = y;
        p.ldy = ldy;
        return p;
    }
    int many(const DenseProduct& p, int n) { return f32 ? launch_dense_gemm_f32(p, n, d.gate_up, st) : launch_dense_gemm_t5(p, n, st); }
    int run(DenseProduct p) {
        if (few && dense_gemv_supported(p, rows)) return launch_dense_gemv(p, rows, st);
        return many(p, rows);
    }
    // a product of the stage's row
    int run_staged(DenseProduct p) {
        if (few) {
            p.stage = &sg;
            if (dense_gemv_supported(p, rows)) {
                routed = p.n2 > 0;
                return launch_dense_gemv(p, rows, st);
            }
            p.stage = nullptr;
        }
        RB_TRY(launch_stream_stage(sg, rows, st));
        p.n2 = 0;
        return run(p);
    }

    // ---- mixers: from the stage to their output rows in d.attn
    int bias_mixer(const rotor_b200_decoder_layer& L, const rotor_b200_decoder_run& r, DenseProduct first) {
        const HeadShape s = shape_of(L, d.cfg.eps);
        const int cols = head_cols(s), ldq = dense_ld(cols);
        BiasAttn at = {};
        at.s = s;
        at.qkv = d.qkv;
        at.ld_qkv = ldq;
        at.f32 = f32;
        at.cache = {r.k_cache, r.v_cache, m.c.d_pos, d.cfg.max_seq, seq};
        at.append = seq == 1;
        at.chunk = L.chunk;
        at.window = L.window;
        at.scale = L.scale;
        at.slopes = L.slopes;
        at.sinks = L.sinks;
        at.out = d.attn;
        at.ld_out = dense_ld(mixer_cols(L));
        at.q = f32 ? nullptr : d.q;
        const bool t5 = bias_attn_t5_supported(at, rows);
        first.w = static_cast<const __nv_bfloat16*>(L.qkv);
        first.n = cols;
        first.y = d.qkv;
        first.ldy = ldq;
        DenseProduct fq = first;
        if (t5) {  // prompts: normalisation and cache append in the product's read-back where the head sizes allow
            fq.epilogue = DENSE_QKV;
            fq.shape = s;
            fq.cache = at.cache;
            fq.q = d.q;
            fq.n2 = 0;
        }
        if (t5 && !m.no_fused && dense_gemm_t5_supported(fq, rows)) {
            RB_TRY(launch_stream_stage(sg, rows, st));
            RB_TRY(launch_dense_gemm_t5(fq, rows, st));
        } else {
            RB_TRY(run_staged(first));
            if (!at.append) {
                HeadFinish hf = {};
                hf.s = s;
                hf.qkv = d.qkv;
                hf.ld_qkv = ldq;
                hf.f32 = f32;
                hf.cache = at.cache;
                hf.q = t5 ? d.q : nullptr;
                RB_TRY(launch_head_finish(hf, rows, st));
            }
        }
        return t5 ? launch_bias_attn_t5(at, rows, st) : launch_bias_attn_rows(at, rows, st);
    }

    int latent_mixer(const rotor_b200_decoder_layer& L, const rotor_b200_decoder_run& r, DenseProduct first, bool staged = true) {
        const LatentShape s = latent_of(L, d.cfg.eps);
        const LatentColumns cols = latent_columns(L);
        const int ld_in = dense_ld(cols.all), qd = latent_q(s), W = latent_row(s), vp = up(s.vdim, 8), lda = dense_ld(s.heads * vp);
        first.w = static_cast<const __nv_bfloat16*>(L.in_proj);
        first.n = cols.all;
        first.y = d.qkv;
        first.ldy = ld_in;
        const bool expanded = !f32 && expanded_attn_supported(s, seq) && expand != 0;
        // prompts: the queries are rotated in the read-back of the product that makes them, where the head sizes allow
        auto turning = [&](DenseProduct p) {
            p.epilogue = DENSE_ROPE;
            p.q_cols = s.heads * qd;
            p.rot_at = s.dp;
            p.rot = s.rot == s.rp ? s.rot : 0;
            p.rope = reinterpret_cast<const float2*>(L.rope);
            p.cache = {nullptr, nullptr, m.c.d_pos, d.cfg.max_seq, seq};
            p.q = static_cast<__nv_bfloat16*>(d.lq);
            p.n2 = 0;
            return p;
        };
        bool turned = false;
        if (expanded && !few && !m.no_fused && !L.q_rank && dense_gemm_t5_supported(turning(first), rows)) {
            turned = true;
            if (staged) RB_TRY(launch_stream_stage(sg, rows, st));
            RB_TRY(many(turning(first), rows));
        } else {
            RB_TRY(staged ? run_staged(first) : run(first));
        }
        const float* dkv = L.own_kv ? d.qkv + cols.q : nullptr;
        const float* gate = L.gated ? d.qkv + cols.q + cols.dkv : nullptr;
        const float* q = d.qkv;
        int ldq = ld_in;
        if (L.q_rank) {
            ldq = dense_ld(s.heads * qd);
            DenseProduct p = plain(L.uq, s.heads * qd, L.q_rank, d.qkv, ld_in, d.q_raw, ldq);
            p.x_raw = 1;
            p.x_norm = L.q_norm;
            p.x_eps = d.cfg.eps;
            if (few && dense_gemv_supported(p, rows)) {
                RB_TRY(launch_dense_gemv(p, rows, st));
            } else {
                const int ldc = dense_ld(L.q_rank);
                RB_TRY(launch_rms_rows(d.qkv, ld_in, L.q_rank, L.q_norm, d.cfg.eps, d.cq, ldc, f32, rows, st));
                const DenseProduct uq = plain(L.uq, s.heads * qd, L.q_rank, d.cq, ldc, d.q_raw, ldq);
                turned = expanded && !m.no_fused && dense_gemm_t5_supported(turning(uq), rows);
                RB_TRY(many(turned ? turning(uq) : uq, rows));
            }
            q = d.q_raw;
        }
        const LatentCache cache = {r.k_cache, m.c.d_pos, d.cfg.max_seq, seq, reinterpret_cast<const float2*>(L.rope)};
        LatentFinish fin = {};
        fin.s = s;
        fin.cache = cache;
        fin.f32 = f32;
        fin.ldq = ldq;
        fin.dkv = dkv;
        fin.ld_dkv = ld_in;
        fin.dkv_norm = L.kv_norm;
        fin.q_out = d.lq;
        if (expanded) {
            fin.q = turned ? nullptr : q;
            RB_TRY(launch_latent_finish(fin, rows, st));
            const int first_pos = L.window > 0 && m.past - L.window + 1 > 0 ? m.past - L.window + 1 : 0, len = m.past + seq - first_pos;
            const int cols_kv = s.heads * (s.dp + vp), step = d.kv_rows / len;
            RB_REQUIRE(step >= 1);
            for (int b0 = 0; b0 < batch; b0 += step) {
                const int nb = batch - b0 < step ? batch - b0 : step;
                __nv_bfloat16* rows0 = static_cast<__nv_bfloat16*>(r.k_cache) + (size_t)b0 * d.cfg.max_seq * W;
                DenseProduct p = product(L.uk_uv, cols_kv, s.rank, rows0 + (size_t)first_pos * W, W);
                p.epilogue = DENSE_HALF;
                p.a = d.kv;
                p.lda = cols_kv;
                p.groups = nb;
                p.gx_row = d.cfg.max_seq;
                p.gy_row = len;
                RB_TRY(launch_dense_gemm_t5(p, len, st));
                ExpandedAttn at = {};
                at.s = s;
                at.cache = cache;
                at.cache.rows = rows0;
                at.cache.past_len += b0;
                at.q = static_cast<const __nv_bfloat16*>(d.lq) + (size_t)b0 * seq * s.heads * qd;
                at.kv = d.kv;
                at.first = first_pos;
                at.len = len;
                at.window = L.window;
                at.scale = L.scale;
                at.sinks = L.sinks;
                at.gate = gate ? gate + (size_t)b0 * seq * ld_in : nullptr;
                at.ld_gate = ld_in;
                at.out = static_cast<__nv_bfloat16*>(d.attn) + (size_t)b0 * seq * lda;
                at.ld_out = lda;
                RB_TRY(launch_expanded_attn(at, nb, st));
            }
            return ROTOR_B200_OK;
        }
        RB_REQUIRE(rows <= d.abs_rows && expand != 1);
        const __nv_bfloat16* uv = static_cast<const __nv_bfloat16*>(L.uk_uv) + (size_t)s.heads * s.dp * dense_ld(s.rank);
        DenseProduct pk = product(L.uk_t, s.kp, s.dim, q, ldq), pv = product(uv, vp, s.rank, d.o_lat, s.heads * s.kp);
        pk.epilogue = pv.epilogue = DENSE_HALF;
        pk.groups = pv.groups = s.heads;
        pk.x_raw = 1;
        pk.gx_col = qd;
        pk.gw_row = s.kp;
        pk.a = d.q_abs;
        pk.lda = s.heads * W;
        pk.gy_col = W;
        pv.gx_col = s.kp;
        pv.gw_row = vp;
        pv.a = d.attn;
        pv.lda = lda;
        pv.gy_col = vp;
        pv.head_gate = gate;
        pv.ld_head_gate = ld_in;
        LatentAttn at = {};
        at.s = s;
        at.cache = cache;
        at.f32 = f32;
        at.q_abs = d.q_abs;
        at.window = L.window;
        at.scale = L.scale;
        at.sinks = L.sinks;
        at.out = d.o_lat;
        if (few && dense_gemv_supported(pk, rows)) {
            if (seq == 1) {  // (the attention kernel makes and appends the token's cache row)
                at.dkv = dkv;
                at.ld_dkv = ld_in;
                at.dkv_norm = L.kv_norm;
                at.early = 1;
            } else {
                RB_TRY(launch_latent_finish(fin, rows, st));
            }
            at.q_raw = q;
            at.ldq = ldq;
            RB_TRY(launch_dense_gemv(pk, rows, st));
        } else {
            fin.q = q;
            fin.q_abs = d.q_abs;
            RB_TRY(launch_latent_finish(fin, rows, st));
            pk.x = d.lq;
            pk.ldx = s.heads * qd;
            pk.x_raw = 0;
            RB_TRY(many(pk, rows));
        }
        RB_TRY(launch_latent_attn(at, rows, st));
        return run(pv);
    }

    // ---- feed-forwards on the normed rows h: the next stage adds what they leave
    int dense_ff(const rotor_b200_decoder_layer& L, const void* h, bool staged, float* y) {
        const int ldf = dense_ld(L.ff);
        DenseProduct up = product(L.gate_up, L.ff, d.cfg.width, h, d.ld);
        up.epilogue = DENSE_GATED;
        up.act = L.act;
        up.a = d.act;
        up.lda = ldf;
        RB_TRY(staged ? run_staged(up) : run(up));
        return run(plain(L.down, d.cfg.width, L.ff, d.act, ldf, y, d.ld));
    }

    int experts_ff(const rotor_b200_decoder_layer& L, const void* h, float* y, StreamStage* next) {
        const int lde = dense_ld(L.experts), ldf = dense_ld(L.ff);
        Routing rt = d.route;
        rt.early = routed;  // (by the input product: the mixer's launches lie between)
        if (!routed) RB_TRY(run(plain(L.router, L.experts, d.cfg.width, h, d.ld, d.logits, lde)));
        routed = false;
        rt.logits = d.logits;
        rt.bias = L.router_b;
        rt.ld = lde;
        rt.experts = L.experts;
        rt.top = L.top;
        DenseProduct up = product(L.gate_up, L.ff, d.cfg.width, h, d.ld), down = plain(L.down, d.cfg.width, L.ff, d.act, ldf, y, d.ld);
        up.epilogue = DENSE_GATED;
        up.act = L.act;
        up.a = d.act;
        up.lda = ldf;
        up.route = down.route = &rt;
        if (few && dense_gemv_supported(up, rows) && dense_gemv_supported(down, rows)) {
            RB_TRY(launch_dense_gemv(up, rows, st));
            return launch_dense_gemv(down, rows, st);
        }
        RB_TRY(launch_route(rt, rows, h, (size_t)d.ld * (f32 ? 4 : 2), d.perm, st));
        up.x = d.perm;
        RB_TRY(many(up, rows * L.top));
        down.epilogue = DENSE_HALF;
        down.a = d.slots;
        down.lda = d.ld;
        RB_TRY(many(down, rows * L.top));
        next->slots = d.slots;
        next->slots_f32 = f32;
        next->slot_of = rt.slot_of;
        next->slot_w = rt.weight;
        next->top = L.top;
        return ROTOR_B200_OK;
    }

    int layer(const rotor_b200_decoder_run& r) {
        const rotor_b200_decoder_layer& L = d.layers[r.layer];
        const bool both = L.parallel && L.ff;
        stage(L.hc1_in, L.norm1, L.norm1_b);
        DenseProduct first = product(nullptr, 0, d.cfg.width, d.h, d.ld);
        if (both) {
            sg.norm2 = L.norm2;
            sg.norm2_b = L.norm2_b;
            sg.h2 = d.h2;
            if (L.experts) {
                first.w2 = static_cast<const __nv_bfloat16*>(L.router);
                first.n2 = L.experts;
                first.y2 = d.logits;
                first.ldy2 = dense_ld(L.experts);
            }
        }
        RB_TRY(is_latent(L) ? latent_mixer(L, r, first) : bias_mixer(L, r, first));
        after(L.hc1_mix, L.hc1_out);
        RB_TRY(run(plain(L.o, d.cfg.width, mixer_cols(L), d.attn, dense_ld(mixer_cols(L)), d.y, d.ld)));
        if (both) {
            sg.y2 = d.y2;
            if (!L.experts) return dense_ff(L, d.h2, false, d.y2);
            RB_TRY(experts_ff(L, d.h2, d.y2, &sg));
            if (sg.slots) sg.y2 = nullptr;
            return ROTOR_B200_OK;
        }
        if (!L.ff) return ROTOR_B200_OK;
        stage(L.hc2_in, L.norm2, L.norm2_b);
        if (!L.experts) {
            RB_TRY(dense_ff(L, d.h, true, d.y));
            after(L.hc2_mix, L.hc2_out);
            return ROTOR_B200_OK;
        }
        RB_TRY(launch_stream_stage(sg, rows, st));
        after(L.hc2_mix, L.hc2_out);
        RB_TRY(experts_ff(L, d.h, d.y, &sg));
        if (sg.slots) sg.y = nullptr;
        return ROTOR_B200_OK;
    }
};

static int run_decoder(Model& m, const long long* ids, int batch, int seq, int logits_mode, float* logits, long long* next_ids,
                cudaStream_t st, bool advance) {
    DecoderStack& d = *m.decoder;
    const rotor_b200_decoder_config& c = d.cfg;
    DecoderPass pass(m, d, batch, seq, st);
    const int rows = pass.rows;
    pass.sg.ids = ids;
    for (const rotor_b200_decoder_run& run : d.runs) RB_TRY(pass.layer(run));
    if (logits_mode == ROTOR_B200_LOGITS_NONE && !next_ids) return ROTOR_B200_OK;

    // sum of the streams and final norm on the rows whose logits are wanted
    const bool all = logits_mode == ROTOR_B200_LOGITS_ALL;
    int lm_rows = rows;
    pass.stage(nullptr, d.final_norm, c.final_norm_b);
    StreamStage& sg = pass.sg;
    sg.x_out = nullptr;
    sg.h = d.hn;
    sg.ldh = d.ldh;
    sg.h_f32 = 1;
    if (m.want || (!all && seq > 1)) {
        d.host_map.clear();
        if (m.want)
            d.host_map.assign(m.want, m.want + m.nwant);
        else
            for (int b = 0; b < batch; ++b) d.host_map.push_back(b * seq + (m.last_of ? m.last_of[b] : seq) - 1);
        lm_rows = (int)d.host_map.size();
        if (!lm_rows) return ROTOR_B200_OK;
        RB_CUDA(cudaMemcpyAsync(d.row_map, d.host_map.data(), d.host_map.size() * sizeof(int), cudaMemcpyHostToDevice, st));
        sg.row_map = d.row_map;
    }
    RB_TRY(launch_stream_stage(sg, lm_rows, st));
    LmHeadParams lp = {};
    lp.embed = d.head;
    lp.x = d.hn;
    lp.xsplit = m.xsplit;
    lp.vocab = c.vocab_size;
    lp.d = d.ldh;
    lp.logits = logits_mode == ROTOR_B200_LOGITS_NONE ? nullptr : logits;
    lp.part_val = m.part_val;
    lp.part_idx = m.part_idx;
    lp.argmax_out = m.want || (all && seq > 1) ? nullptr : next_ids;
    lp.nparts = lmhead_parts();
    lp.tail_counter = m.c.counters + 3;
    if (advance) {
        lp.adv_log = m.tok_log;
        lp.adv_pos = m.c.d_pos;
        lp.adv_step = m.d_step;
        lp.adv_max_log = m.max_log;
    }
    return launch_lmhead(lp, lm_rows, st);
}

static void destroy_decoder(Model& m) { delete m.decoder; }
static const ModelFamily DECODER_FAMILY = {run_decoder, destroy_decoder};

}  // namespace rb

using namespace rb;

extern "C" {

size_t rotor_b200_decoder_workspace_bytes(const rotor_b200_decoder_config* cfg, const rotor_b200_decoder_layer* layers) {
    if (!cfg || !layers || check_decoder(*cfg, layers, nullptr)) return 0;
    Model m;
    memset(&m, 0, sizeof(m));
    DecoderStack d;
    d.cfg = *cfg;
    d.absorb_all = false;
    size_t total = 0;
    carve_decoder(m, d, layers, nullptr, &total);
    return total;
}

int rotor_b200_decoder_create(const rotor_b200_decoder_config* cfg, const rotor_b200_decoder_layer* layers,
                              const rotor_b200_decoder_run* runs, const void* embed, const void* head, const float* final_norm,
                              void* workspace, size_t workspace_bytes, void** handle) {
    RB_REQUIRE(cfg && layers && runs && embed && head && final_norm && workspace && handle);
    RB_REQUIRE(((uintptr_t)workspace & 255) == 0);
    int rc = check_decoder(*cfg, layers, runs);
    if (rc) return rc;
    for (int l = 0; l < cfg->n_layers; ++l) {
        const rotor_b200_decoder_layer& L = layers[l];
        RB_REQUIRE(L.o && L.norm1 && L.hc1_in && L.hc1_mix && L.hc1_out);
        RB_REQUIRE(is_latent(L) ? L.in_proj && L.uk_uv && L.uk_t && L.rope && (!L.own_kv || L.kv_norm) && (!L.q_rank || (L.uq && L.q_norm))
                                : L.qkv != nullptr);
        RB_REQUIRE(!L.ff || (L.gate_up && L.down && L.norm2 && (!L.experts || L.router)));
        RB_REQUIRE(!L.ff || L.parallel || (L.hc2_in && L.hc2_mix && L.hc2_out));
    }
    Model* m = new (std::nothrow) Model;
    DecoderStack* d = new (std::nothrow) DecoderStack;
    if (!m || !d) {
        delete m;
        delete d;
        return ROTOR_B200_ERR_ARG;
    }
    memset(m, 0, sizeof(*m));
    m->family = &DECODER_FAMILY;
    m->decoder = d;
    m->no_fused = getenv("ROTOR_B200_NO_FUSED_STEP") != nullptr;
    d->cfg = *cfg;
    d->absorb_all = false;
    d->layers.assign(layers, layers + cfg->n_layers);
    d->runs.assign(runs, runs + cfg->n_runs);
    d->embed = static_cast<const __nv_bfloat16*>(embed);
    d->head = static_cast<const __nv_bfloat16*>(head);
    d->final_norm = final_norm;
    // what the shared entry points read of the configuration
    m->cfg.vocab_size = cfg->vocab_size;
    m->cfg.d_model = cfg->width;
    m->cfg.n_layers = cfg->n_runs;
    m->cfg.causal = 1;
    m->cfg.max_batch = cfg->max_batch;
    m->cfg.max_seq = cfg->max_seq;
    m->cfg.max_rows = cfg->max_rows;
    m->c.max_batch = cfg->max_batch;
    m->c.max_seq = cfg->max_seq;
    size_t total = 0;
    carve_decoder(*m, *d, layers, static_cast<unsigned char*>(workspace), &total);
    rc = total > workspace_bytes ? ROTOR_B200_ERR_WORKSPACE : ROTOR_B200_OK;
    // pad columns of activations stay zero from here on (or hold other products' finite values)
    if (!rc && cudaMemset(workspace, 0, total) != cudaSuccess) rc = ROTOR_B200_ERR_CUDA;
    if (!rc) rc = configure_lmhead();
    if (!rc) rc = configure_dense();
    if (!rc && cudaDeviceSynchronize() != cudaSuccess) rc = ROTOR_B200_ERR_CUDA;
    if (rc) {
        delete d;
        delete m;
        return rc;
    }
    *handle = m;
    return ROTOR_B200_OK;
}

int rotor_b200_stream_stage(const int64_t* ids, const void* embed, int vocab, const float* x_in, float* x_out, const float* y,
                            const float* mix, const float* out, const float* in, const float* norm, float eps, int rows,
                            int streams, int n, void* h, int h_f32, void* stream) {
    RB_REQUIRE(rows > 0 && n > 0 && streams >= 1 && streams <= STREAMS_MAX && (!h || norm));
    RB_REQUIRE(ids ? embed != nullptr && vocab > 0 : x_in && y && mix && out && x_in != x_out);
    StreamStage p = {};
    p.streams = streams;
    p.n = n;
    p.ld = p.ldh = dense_ld(n);
    p.ids = (const long long*)ids;
    p.embed = static_cast<const __nv_bfloat16*>(embed);
    p.vocab = vocab;
    p.embed_scale = 1.f;
    p.x_in = x_in;
    p.x_out = x_out;
    p.y = y;
    p.mix = mix;
    p.out = out;
    p.in = in;
    p.norm = norm;
    p.eps = eps;
    p.h = h;
    p.h_f32 = h_f32;
    return launch_stream_stage(p, rows, as_stream(stream));
}

int rotor_b200_dense_linear(const void* w, int n, int k, const void* x, int rows, int f32, int gated, void* y, float* scratch,
                            void* stream) {
    RB_REQUIRE(w && x && y && n > 0 && k > 0 && rows > 0);
    DenseProduct p = {};
    p.w = static_cast<const __nv_bfloat16*>(w);
    p.n = n;
    p.k = k;
    p.ldw = p.ldx = dense_ld(k);
    p.f32 = f32;
    p.x = x;
    p.epilogue = gated ? DENSE_GATED : DENSE_PLAIN;
    if (gated) {
        p.a = y;
        p.lda = dense_ld(n);
    } else {
        p.y = static_cast<float*>(y);
        p.ldy = dense_ld(n);
    }
    RB_TRY(configure_dense());
    cudaStream_t st = as_stream(stream);
    if (dense_gemv_supported(p, rows)) return launch_dense_gemv(p, rows, st);
    return f32 ? launch_dense_gemm_f32(p, rows, scratch, st) : launch_dense_gemm_t5(p, rows, st);
}

int rotor_b200_norm_stage(const int64_t* ids, const void* embed, int vocab, float embed_scale, const float* x_in, float* x_out,
                          const float* y, const float* y2, const float* norm, const float* norm_b, const float* norm2,
                          const float* norm2_b, float eps, int rows, int n, void* h, void* h2, int h_f32, void* stream) {
    RB_REQUIRE(rows > 0 && n > 0 && norm && h && (ids ? embed != nullptr && vocab > 0 : x_in && x_in != x_out));
    StreamStage p = {};
    p.streams = 1;
    p.n = n;
    p.ld = p.ldh = dense_ld(n);
    p.ids = (const long long*)ids;
    p.embed = static_cast<const __nv_bfloat16*>(embed);
    p.vocab = vocab;
    p.embed_scale = embed_scale;
    p.x_in = x_in;
    p.x_out = x_out;
    p.y = y;
    p.y2 = y2;
    p.norm = norm;
    p.norm_b = norm_b;
    p.norm2 = norm2;
    p.norm2_b = norm2_b;
    p.eps = eps;
    p.h = h;
    p.h2 = h2;
    p.h_f32 = h_f32;
    return launch_stream_stage(p, rows, as_stream(stream));
}

// A stack of one layer over a caller's workspace, for the entry points of single sublayers.
struct OneLayer {
    Model m;
    DecoderStack d;
    int set(const rotor_b200_decoder_config* cfg, const rotor_b200_decoder_layer* layer, void* workspace, size_t bytes) {
        memset(&m, 0, sizeof(m));
        RB_REQUIRE(cfg && layer && workspace && ((uintptr_t)workspace & 255) == 0 && cfg->n_layers == 1);
        RB_TRY(check_decoder(*cfg, layer, nullptr));
        d.cfg = *cfg;
        d.absorb_all = true;
        m.decoder = &d;
        m.no_fused = getenv("ROTOR_B200_NO_FUSED_STEP") != nullptr;
        size_t total = 0;
        carve_decoder(m, d, layer, static_cast<unsigned char*>(workspace), &total);
        return total > bytes ? ROTOR_B200_ERR_WORKSPACE : configure_dense();
    }
};

size_t rotor_b200_decoder_layer_workspace_bytes(const rotor_b200_decoder_config* cfg, const rotor_b200_decoder_layer* layer) {
    if (!cfg || !layer || cfg->n_layers != 1 || check_decoder(*cfg, layer, nullptr)) return 0;
    Model m;
    memset(&m, 0, sizeof(m));
    DecoderStack d;
    d.cfg = *cfg;
    d.absorb_all = true;
    size_t total = 0;
    carve_decoder(m, d, layer, nullptr, &total);
    return total;
}

int rotor_b200_latent_mixer(const rotor_b200_decoder_config* cfg, const rotor_b200_decoder_layer* layer, const void* h, int batch,
                            int seq, int past, void* cache, int expanded, float* y, void* workspace, size_t workspace_bytes,
                            void* stream) {
    OneLayer one;
    RB_TRY(one.set(cfg, layer, workspace, workspace_bytes));
    RB_REQUIRE(is_latent(*layer) && h && cache && y && batch > 0 && seq > 0 && past >= 0 && past + seq <= cfg->max_seq);
    RB_REQUIRE(batch <= cfg->max_batch && batch * seq <= cfg->max_rows && layer->in_proj && layer->uk_uv && layer->uk_t && layer->o && layer->rope);
    cudaStream_t st = as_stream(stream);
    RB_TRY(launch_set_pos(one.m.c.d_pos, cfg->max_batch, past, nullptr, st));
    one.m.past = past;
    DecoderPass pass(one.m, one.d, batch, seq, st);
    pass.expand = expanded;
    const rotor_b200_decoder_run run = {0, cache, nullptr};
    RB_TRY(pass.latent_mixer(*layer, run, pass.product(nullptr, 0, cfg->width, h, one.d.ld), false));
    return pass.run(pass.plain(layer->o, cfg->width, mixer_cols(*layer), one.d.attn, dense_ld(mixer_cols(*layer)), y, one.d.ld));
}

int rotor_b200_experts(const rotor_b200_decoder_config* cfg, const rotor_b200_decoder_layer* layer, const void* h, int rows,
                       float* y, void* workspace, size_t workspace_bytes, void* stream) {
    OneLayer one;
    RB_TRY(one.set(cfg, layer, workspace, workspace_bytes));
    RB_REQUIRE(layer->experts > 0 && h && y && rows > 0 && rows <= cfg->max_rows && layer->router && layer->gate_up && layer->down);
    cudaStream_t st = as_stream(stream);
    DecoderPass pass(one.m, one.d, rows, 1, st);
    StreamStage sum = pass.sg;
    RB_TRY(pass.experts_ff(*layer, h, y, &sum));
    if (!sum.slots) return ROTOR_B200_OK;
    // the tokens' slots added up by a stage of their own, over a residual of zeros
    RB_CUDA(cudaMemsetAsync(one.d.x[0], 0, (size_t)rows * one.d.ld * sizeof(float), st));
    sum.streams = 1;
    sum.x_in = one.d.x[0];
    sum.x_out = y;
    sum.y = nullptr;
    sum.h = nullptr;
    return launch_stream_stage(sum, rows, st);
}

int rotor_b200_bias_attention(const rotor_b200_decoder_layer* layer, float eps, int f32, const float* qkv, int batch, int seq,
                              const int32_t* past_len, int max_seq, void* k_cache, void* v_cache, void* out, int row_kernel,
                              void* q_scratch, void* stream) {
    RB_REQUIRE(layer && qkv && past_len && k_cache && v_cache && out && batch > 0 && seq > 0 && max_seq > 0);
    RB_REQUIRE(layer->heads > 0 && layer->kv_heads > 0 && layer->heads % layer->kv_heads == 0 && layer->dim > 0 && layer->vdim > 0);
    cudaStream_t st = as_stream(stream);
    const HeadShape s = shape_of(*layer, eps);
    const CacheView cache = {k_cache, v_cache, past_len, max_seq, seq};
    BiasAttn at = {};
    at.s = s;
    at.qkv = qkv;
    at.ld_qkv = dense_ld(head_cols(s));
    at.f32 = f32;
    at.q = row_kernel || f32 ? nullptr : static_cast<const __nv_bfloat16*>(q_scratch);
    at.cache = cache;
    at.append = seq == 1;
    at.chunk = layer->chunk;
    at.window = layer->window;
    at.scale = layer->scale;
    at.slopes = layer->slopes;
    at.sinks = layer->sinks;
    at.out = out;
    at.ld_out = dense_ld(s.heads * s.vdim);
    const int rows = batch * seq;
    const bool t5 = bias_attn_t5_supported(at, rows);
    if (!at.append) {
        HeadFinish hf = {};
        hf.s = s;
        hf.qkv = qkv;
        hf.ld_qkv = at.ld_qkv;
        hf.f32 = f32;
        hf.cache = cache;
        hf.q = t5 ? static_cast<__nv_bfloat16*>(q_scratch) : nullptr;
        RB_TRY(launch_head_finish(hf, rows, st));
    }
    return t5 ? launch_bias_attn_t5(at, rows, st) : launch_bias_attn_rows(at, rows, st);
}

}  // extern "C"

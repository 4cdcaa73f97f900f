// Driver of layer-described decoders: a list of layer runs (a layer may run several times in a row with
// the same weights, each run with its own cache), residual streams with hyper-connections, bias / chunk
// attention, gated feed-forward, an output head of its own.  It sits behind the same model handle as the
// ternary model: position state, generation loop, token log and captured graph are handle.cu's.
//
// Launch sequence of a forward, per layer run
//   many rows:  stage (streams, norm) -> q/k/v product [-> head finish] -> attention -> o product
//               -> stage -> gate/up product (gating in its read-back) -> down product
//   up to DENSE_FEW_ROWS rows: the stages ride in the q/k/v and gate/up products' prologues; a generation
//               step's attention kernel normalises and appends its own row: five launches per run
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
    float* y;                    // sublayer output [rows][ld]
    void* h;                     // sublayer input [rows][ld]
    float* qkv;                  // raw projections
    __nv_bfloat16* q;            // normalised queries
    void* attn;                  // attention rows
    void* act;                   // gated rows
    float* gate_up;              // float32 runs: both halves before the gating
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
    }
    if (runs)
        for (int r = 0; r < c.n_runs; ++r)
            if (runs[r].layer < 0 || runs[r].layer >= c.n_layers || !runs[r].k_cache || !runs[r].v_cache) return ROTOR_B200_ERR_ARG;
    return ROTOR_B200_OK;
}

static void carve_decoder(Model& m, DecoderStack& d, const rotor_b200_decoder_layer* layers, unsigned char* base, size_t* total) {
    const rotor_b200_decoder_config& c = d.cfg;
    const size_t rows = c.max_rows, esz = c.f32 ? 4 : 2;
    size_t qkv = 0, q = 0, attn = 0, act = 0, gu = 0;
    for (int l = 0; l < c.n_layers; ++l) {
        const HeadShape s = shape_of(layers[l], c.eps);
        const size_t a[5] = {(size_t)dense_ld(head_cols(s)), (size_t)s.heads * s.kd, (size_t)dense_ld(s.heads * s.vdim),
                             (size_t)dense_ld(layers[l].ff), (size_t)2 * layers[l].ff};
        qkv = a[0] > qkv ? a[0] : qkv;
        q = a[1] > q ? a[1] : q;
        attn = a[2] > attn ? a[2] : attn;
        act = a[3] > act ? a[3] : act;
        gu = a[4] > gu ? a[4] : gu;
    }
    d.ld = dense_ld(c.width);
    d.ldh = (c.width + 255) / 256 * 256;
    Carve cv{base, 0};
    for (int i = 0; i < 2; ++i) d.x[i] = cv.take<float>(rows * c.streams * d.ld);
    d.y = cv.take<float>(rows * d.ld);
    d.h = cv.take<unsigned char>(rows * d.ld * esz);
    d.qkv = cv.take<float>(rows * qkv);
    d.q = cv.take<__nv_bfloat16>(c.f32 ? 1 : rows * q);
    d.attn = cv.take<unsigned char>(rows * attn * esz);
    d.act = cv.take<unsigned char>((rows * act + 1) * esz);
    d.gate_up = cv.take<float>(c.f32 ? rows * gu + 1 : 1);
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

static int run_decoder(Model& m, const long long* ids, int batch, int seq, int logits_mode, float* logits, long long* next_ids,
                cudaStream_t st, bool advance) {
    DecoderStack& d = *m.decoder;
    const rotor_b200_decoder_config& c = d.cfg;
    const int rows = batch * seq, f32 = c.f32;
    const bool few = rows <= DENSE_FEW_ROWS && !m.no_fused;
    int cur = 0;  // buffer the next stage writes
    StreamStage sg = {};
    sg.streams = c.streams;
    sg.n = c.width;
    sg.ld = d.ld;
    sg.ids = ids;
    sg.embed = d.embed;
    sg.vocab = c.vocab_size;
    sg.eps = c.eps;
    sg.y = d.y;
    sg.h = d.h;
    sg.ldh = d.ld;
    sg.h_f32 = f32;
    // points the stage at the sublayer that follows; the caller runs it
    auto stage = [&](const float* in, const float* norm) {
        sg.in = in;
        sg.norm = norm;
        sg.x_in = d.x[cur ^ 1];
        sg.x_out = d.x[cur];
    };
    // after the stage has run: the coefficients of the sublayer whose output the next stage adds
    auto after = [&](const float* mix, const float* out) {
        sg.ids = nullptr;
        sg.mix = mix;
        sg.out = out;
        cur ^= 1;
    };
    auto product = [&](const void* w, int n, int k, const void* x, int ldx, bool with_stage, int epi, float* y, int ldy, void* a,
                       int lda) {
        DenseProduct p = {};
        p.w = static_cast<const __nv_bfloat16*>(w);
        p.n = n;
        p.k = k;
        p.ldw = dense_ld(k);
        p.f32 = f32;
        p.x = x;
        p.ldx = ldx;
        p.epilogue = epi;
        p.y = y;
        p.ldy = ldy;
        p.a = a;
        p.lda = lda;
        if (few && dense_gemv_supported(p, rows)) {
            p.stage = with_stage ? &sg : nullptr;
            return launch_dense_gemv(p, rows, st);
        }
        if (with_stage) {
            const int rc = launch_stream_stage(sg, rows, st);
            if (rc) return rc;
        }
        return f32 ? launch_dense_gemm_f32(p, rows, d.gate_up, st) : launch_dense_gemm_t5(p, rows, st);
    };

    for (const rotor_b200_decoder_run& run : d.runs) {
        const rotor_b200_decoder_layer& L = d.layers[run.layer];
        const HeadShape s = shape_of(L, c.eps);
        const int cols = head_cols(s), ldq = dense_ld(cols), lda = dense_ld(s.heads * s.vdim);
        const CacheView cache = {run.k_cache, run.v_cache, m.c.d_pos, c.max_seq, seq};
        BiasAttn at = {};
        at.s = s;
        at.qkv = d.qkv;
        at.ld_qkv = ldq;
        at.f32 = f32;
        at.cache = cache;
        at.append = seq == 1;
        at.chunk = L.chunk;
        at.scale = L.scale;
        at.slopes = L.slopes;
        at.out = d.attn;
        at.ld_out = lda;
        at.q = f32 ? nullptr : d.q;
        const bool t5 = bias_attn_t5_supported(at, rows);

        stage(L.hc1_in, L.norm1);
        DenseProduct fq = {};
        if (t5) {  // prompts: normalisation and cache append in the product's read-back where the head sizes allow
            fq.w = static_cast<const __nv_bfloat16*>(L.qkv);
            fq.n = cols;
            fq.k = c.width;
            fq.ldw = d.ld;
            fq.x = d.h;
            fq.ldx = d.ld;
            fq.epilogue = DENSE_QKV;
            fq.shape = s;
            fq.cache = cache;
            fq.q = d.q;
        }
        if (t5 && !m.no_fused && dense_gemm_t5_supported(fq, rows)) {
            RB_TRY(launch_stream_stage(sg, rows, st));
            RB_TRY(launch_dense_gemm_t5(fq, rows, st));
        } else {
            RB_TRY(product(L.qkv, cols, c.width, d.h, d.ld, true, DENSE_PLAIN, d.qkv, ldq, nullptr, 0));
            if (!at.append) {
                HeadFinish hf = {};
                hf.s = s;
                hf.qkv = d.qkv;
                hf.ld_qkv = ldq;
                hf.f32 = f32;
                hf.cache = cache;
                hf.q = t5 ? d.q : nullptr;
                RB_TRY(launch_head_finish(hf, rows, st));
            }
        }
        after(L.hc1_mix, L.hc1_out);
        RB_TRY(t5 ? launch_bias_attn_t5(at, rows, st) : launch_bias_attn_rows(at, rows, st));
        RB_TRY(product(L.o, c.width, s.heads * s.vdim, d.attn, lda, false, DENSE_PLAIN, d.y, d.ld, nullptr, 0));
        if (!L.ff) continue;
        const int ldf = dense_ld(L.ff);
        stage(L.hc2_in, L.norm2);
        RB_TRY(product(L.gate_up, L.ff, c.width, d.h, d.ld, true, DENSE_GATED, nullptr, 0, d.act, ldf));
        after(L.hc2_mix, L.hc2_out);
        RB_TRY(product(L.down, c.width, L.ff, d.act, ldf, false, DENSE_PLAIN, d.y, d.ld, nullptr, 0));
    }
    if (logits_mode == ROTOR_B200_LOGITS_NONE && !next_ids) return ROTOR_B200_OK;

    // sum of the streams and final norm on the rows whose logits are wanted
    const bool all = logits_mode == ROTOR_B200_LOGITS_ALL;
    int lm_rows = rows;
    stage(nullptr, d.final_norm);
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
        RB_REQUIRE(L.qkv && L.o && L.norm1 && L.hc1_in && L.hc1_mix && L.hc1_out);
        RB_REQUIRE(!L.ff || (L.gate_up && L.down && L.norm2 && L.hc2_in && L.hc2_mix && L.hc2_out));
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
    static PerDevice<bool> once;
    if (!once.here()) {
        RB_TRY(configure_dense());
        once.here() = true;
    }
    cudaStream_t st = as_stream(stream);
    if (dense_gemv_supported(p, rows)) return launch_dense_gemv(p, rows, st);
    return f32 ? launch_dense_gemm_f32(p, rows, scratch, st) : launch_dense_gemm_t5(p, rows, st);
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
    at.scale = layer->scale;
    at.slopes = layer->slopes;
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

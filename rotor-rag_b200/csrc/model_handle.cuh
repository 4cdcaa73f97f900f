// State behind a model handle, shared by the drivers of the model families (model.cu: the ternary
// model; decoder.cu: decoders described layer by layer).  The generation loop, its token log and its
// captured graph (handle.cu) work on this state whatever the family.
#pragma once
#include "model.cuh"

namespace rb {

#define RB_TRY(expr)              \
    do {                          \
        int rc_ = (expr);         \
        if (rc_) return rc_;      \
    } while (0)

inline size_t al256(size_t v) { return (v + 255) & ~(size_t)255; }

struct Model;
struct DecoderStack;

// What a family supplies.  forward: one forward over ids (device [batch * seq]); cached lengths are read
// from m.c.d_pos; logits of the last positions, of all, or of the rows m.want; with `advance` the call is a
// generation step that also logs its picks and moves the positions on.
struct ModelFamily {
    int (*forward)(Model& m, const long long* ids, int batch, int seq, int logits_mode, float* logits,
                   long long* next_ids, cudaStream_t st, bool advance);
    void (*destroy)(Model& m);
};

// Scratch buffers and dimensions one block needs; carved from caller-owned device memory.
struct Ctx {
    int d, ff, n_heads, n_kv_heads, head_dim, dq, dkv;
    int terms, ffn_act, causal, variant, max_seq;
    float rope_theta, eps;
    size_t kmax;  // widest padded BitLinear input
    float* h;     // residual stream [rows][d]
    float* h2;    // second copy: fused generation steps ping-pong between the two
    float* hn;    // final-normed rows
    float* qbuf;
    float* attn;
    int8_t* xq;
    float* sx[2];
    int32_t* xsum[2];
    int32_t* accA;  // q/k/v and gate/up accumulators
    int32_t* accB;  // o and down accumulators
    int* d_pos;
    float2* rope;        // cos/sin table, or null
    float2* rope_buf;    // storage for it
    __nv_bfloat16* kvsplit;  // prefill attention: hi / lo bf16 planes of one layer's K/V rows (or null)
    size_t kvsplit_plane;
    float* part_o;       // decode-attention partials
    float* part_m;
    float* part_l;
    int nsplit;
    int max_batch;
    unsigned* counters;  // [8 + max_batch] zeroed words for last-CTA tails
    // tensor parallel (tp_size > 1): communicator, whole FFN width, exchange buffers
    void* tp;
    int tp_size, ff_total;
    float* stat[2];      // [rows] per-row statistics that cross ranks (sum of squares, absolute maximum)
    float* gated;        // [rows][ff] this rank's slice of the gated FFN row
    // float32 outputs of the fused generation step's products: q/k/v, o, gated, down
    float* fy[4];
};

constexpr int FUSED_MAX_ROWS = 4;

struct Model {
    const ModelFamily* family;
    rotor_b200_model_config cfg;
    rotor_b200_layer_weights* layers;
    const __nv_bfloat16* embed;
    const float* final_norm;
    Ctx c;
    float* part_val;
    int* part_idx;
    long long* cur_ids;
    long long* tok_log;
    int* d_step;
    int* d_lens;                // [max_batch] prompt lengths of a ragged batch
    const int32_t* last_of;     // host, during a ragged forward: tokens of each sequence (its last row is picked)
    int max_log;
    // host mirror of the generation state
    int pos, step, batch;
    cudaGraphExec_t graph;
    int graph_batch;
    unsigned long long graph_launches;  // kernels inside the captured step
    // tensor parallel greedy pick: (value, global index) of every rank's best row
    __nv_bfloat16* xsplit;  // LM head over more than four rows: hi / lo bf16 split of its input rows
    float* pick_val;      // [rows]
    long long* pick_idx;  // [rows]
    unsigned char* pick_send;  // [rows] x 12 bytes
    unsigned char* pick_recv;  // [tp][rows] x 12 bytes
    // layer-described decoder (decoder.cu): its stack of layers, or null for the ternary model
    DecoderStack* decoder;
    bool no_fused;        // comparison aid: unfused stages in every forward
    const int32_t* want;  // host, during a forward of selected rows: rows whose logits are wanted
    int nwant;
    int past;             // during a forward of many tokens: their sequences' cached length
};

struct Carve {
    unsigned char* base;
    size_t off;
    template <typename T>
    T* take(size_t count) {
        T* p = base ? reinterpret_cast<T*>(base + off) : nullptr;
        off += al256(count * sizeof(T));
        return p;
    }
};

int launch_set_pos(int* pos, int n, int v, const int* lens, cudaStream_t st);
// logs the picked tokens and moves every position on by one
int launch_advance(Model& m, const long long* picked, int batch, cudaStream_t st);

}  // namespace rb

// Kernels of layer-described decoders: dense bf16 weights, residual streams with hyper-connections,
// attention with normalised queries and keys, a distance bias, chunk and window masks and softmax sinks,
// latent attention, gated feed-forward, routed experts.  Every size and constant is a parameter; a design
// is a choice of them (decoder.cu).
//
// Conventions: activations are bf16, or float32 when `f32` is set (then nothing is rounded below
// float32 and no tensor core is used).  Row strides ("ld") are in elements and multiples of 64, the
// pad columns of weights and residual streams are zero.  Weights are bf16 in both modes.
#pragma once
#include <cuda_bf16.h>

#include "model.cuh"

namespace rb {

constexpr int DENSE_LD = 64;       // row strides are multiples of this
constexpr int DENSE_FEW_ROWS = 4;  // up to this many rows a product is a matrix-vector product with its stage fused in
constexpr int STREAMS_MAX = 16;

inline int dense_ld(int n) { return (n + DENSE_LD - 1) / DENSE_LD * DENSE_LD; }

// Residual stage between two sublayers of a model with `streams` residual streams per token:
//   X_t <- sum_s mix[s][t] X_s + out[t] y        (y: output of the sublayer before; all t from the old X)
//   u    = sum_s in[s] X_s                        (in null: plain sum)
//   h    = u / sqrt(mean(u^2) + eps) * norm       (input of the sublayer that follows)
// One stream with mix = in = out = 1 is the ordinary pre-norm residual.  With norm_b the norm is a layer
// norm, (u - mean) / sqrt(var + eps) * norm + norm_b.  y may be a sum: of y, y2 and the weighted rows a
// token's experts left in `slots` (sublayers that read the same residual); norm2 gives a second normed
// row h2 of the same u.
struct StreamStage {
    int streams, n, ld;          // width and row stride of one stream
    const long long* ids;        // set: X_s <- embed[id] for every s instead of the mix
    const __nv_bfloat16* embed;  // [vocab][ld]
    int vocab;
    float embed_scale;
    const float* x_in;           // [rows][streams][ld]
    float* x_out;                // [rows][streams][ld], not x_in; null: the new streams are not kept
    const float* y;              // [rows][ld], or null
    const float* y2;             // [rows][ld], or null
    const void* slots;           // [slot][ld] expert outputs (float32 or bf16), or null
    const int* slot_of;          // [rows][top]
    const float* slot_w;         // [rows][top]
    int top, slots_f32;
    const float* mix;            // [from][to]
    const float* out;
    const float* in;
    const float* norm;           // [ld]
    const float* norm_b;         // [ld], or null: root mean square norm
    const float* norm2;          // second normed row of the same u, or null
    const float* norm2_b;
    float eps;
    const int* row_map;          // optional: output row r comes from source row row_map[r]
    void* h;                     // [rows][ldh]; columns past n are written as zeros
    void* h2;                    // [rows][ldh], with norm2
    int ldh;
    int h_f32;
};
int launch_stream_stage(const StreamStage& p, int rows, cudaStream_t st);

enum DenseEpilogue { DENSE_PLAIN = 0, DENSE_GATED = 1, DENSE_QKV = 2, DENSE_HALF = 3, DENSE_ROPE = 4 };
enum GateAct { ACT_GELU_TANH = 0, ACT_SILU = 1 };
constexpr int EXPERTS_MAX = 1024, EXPERT_TOP_MAX = 32;

// Which experts the tokens of a call use (experts.cu).  `logits` are the router's raw outputs.
struct Routing {
    const float* logits;         // [rows][ld]
    const float* bias;           // [experts], added to them; or null
    int ld, experts, top;
    int early;                   // the outputs were written two or more launches ago: they may be read before the launch wait
    // many rows: filled by launch_route
    int* slot_of;                // [rows][top] slot of a token's k-th choice; slots of one expert are consecutive
    float* weight;               // [rows][top] softmax over the chosen logits
    int* chosen;                 // [rows][top]
    int* counts;                 // [experts] zeroed words
    int* cursor;                 // [experts]
    int* table;                  // tiles of `tile_rows` slots: count, then (expert, first slot, slots) per tile
    int tile_rows, max_tiles;    // (what counts that were not zeroed could say is cut to the table's size)
};
inline int route_tiles(long long slots, int experts, int tile_rows) { return (int)(slots / tile_rows) + experts; }
// chooses the experts of every row, and copies the rows x (16-byte pieces) into their slots of `permuted`
int launch_route(const Routing& r, int rows, const void* x, size_t row_bytes, void* permuted, cudaStream_t st);

struct HeadShape {
    int heads, kv_heads, dim, vdim;
    int kd, vd;                  // row widths of the caches: dim and vdim rounded up to 8
    int unit;                    // queries and keys are divided by their root mean square over dim
    float eps;
};
inline int head_cols(const HeadShape& s) { return (s.heads + s.kv_heads) * s.dim + s.kv_heads * s.vdim; }

// Where the rows of a call live in the caches: row = sequence * seq + i sits at past_len[sequence] + i.
struct CacheView {
    void* k;                     // [sequence][kv_heads][max_seq][kd]
    void* v;                     // [sequence][kv_heads][max_seq][vd]
    const int* past_len;
    int max_seq, seq;
};

// y[r][o] = sum_k x[r][k] w[o][k].  `groups` > 1: as many products with operands at fixed distances (the heads
// of a per-head product, the sequences of a cache).
struct DenseProduct {
    const __nv_bfloat16* w;      // [n][ldw]; gated: [2 n][ldw], gate rows then up rows
    int n, k, ldw;
    int f32;                     // activation type
    const void* x;               // [rows][ldx]
    int ldx;
    const StreamStage* stage;    // few rows only: x is this stage's output, computed on the way
    // DENSE_PLAIN: y float32; DENSE_GATED: a = act(gate) * up in the activation type; DENSE_HALF: a in the activation
    // type, with head_gate multiplied by sigmoid(head_gate[r][group])
    int epilogue;
    int act;
    float* y;
    int ldy;
    void* a;
    int lda;
    // DENSE_QKV (bf16): rows are [q heads | k heads | v heads]; normalised q rows out, k and v rows appended
    HeadShape shape;
    CacheView cache;
    __nv_bfloat16* q;            // [rows][heads * kd]
    // DENSE_ROPE (bf16): the first q_cols outputs are query heads of rot_at plain and rot columns to be rotated by their
    // token's position, bf16 rows of their own in q; the rest is float32 in y
    int q_cols, rot_at, rot;
    const float2* rope;          // [max_seq][rot / 2]
    // groups (0 means 1): distances in elements (x columns and rows, w rows, output columns and rows)
    int groups, gx_col, gx_row, gw_row, gy_col, gy_row;
    const float* head_gate;
    int ld_head_gate;
    // few rows only.  x_raw: x is float32 whatever the activation type, divided by its root mean square and
    // multiplied by x_norm if given, then rounded to the activation type
    int x_raw;
    const float* x_norm;
    float x_eps;
    // with a stage that has a norm2: a second small product of h2, float32 (n2 = 0: h2 alone)
    const __nv_bfloat16* w2;
    int n2;
    float* y2;
    int ldy2;
    // experts: few rows, gated: row r, choice k -> a[r * top + k]; plain: x holds those rows and y[r] is their
    // weighted sum.  Many rows: the rows of x are slots, and `route` holds the tile table
    const Routing* route;
};
bool dense_gemv_supported(const DenseProduct& p, int rows);
int launch_dense_gemv(const DenseProduct& p, int rows, cudaStream_t st);
bool dense_gemm_t5_supported(const DenseProduct& p, int rows);
int launch_dense_gemm_t5(const DenseProduct& p, int rows, cudaStream_t st);
int launch_dense_gemm_f32(const DenseProduct& p, int rows, float* gate_up, cudaStream_t st);
int configure_dense();

// Raw projection rows -> normalised q rows (optional) and appended k / v cache rows.
struct HeadFinish {
    HeadShape s;
    const float* qkv;            // [rows][ld_qkv]
    int ld_qkv, f32;
    CacheView cache;
    __nv_bfloat16* q;            // [rows][heads * kd], or null
};
int launch_head_finish(const HeadFinish& p, int rows, cudaStream_t st);

// softmax over the visible keys j of  (q . k_j) scale - slope (i - j);  j <= i, j in i's chunk if chunk > 0, and
// i - j < window if window > 0.  A sink adds exp(sink_h) to the denominator of head h.
struct BiasAttn {
    HeadShape s;
    const float* qkv;            // raw projections: queries are normalised on the way (row kernel)
    int ld_qkv, f32;
    const __nv_bfloat16* q;      // normalised queries (tensor-core kernel)
    CacheView cache;
    int append;                  // one token per sequence: its key and value are taken from qkv and appended here
    int chunk, window;
    float scale;
    const float* slopes;         // [heads], or null for no bias
    const float* sinks;          // [heads], or null
    void* out;                   // [rows][ld_out], head h at column h * vdim
    int ld_out;
};
int bias_attn_reach(const BiasAttn& p);  // most keys one query can see
int launch_bias_attn_rows(const BiasAttn& p, int rows, cudaStream_t st);
bool bias_attn_t5_supported(const BiasAttn& p, int rows);
int launch_bias_attn_t5(const BiasAttn& p, int rows, cudaStream_t st);

// Latent attention.  A position's cache row is [latent, rank rounded up to 16 | rotated key part, rot_dim rounded
// up to 16], pads zero; a head's query row is [dim rounded up to 8 | rot rounded up to 16].
//   absorbed: the queries are taken into the latent space (W_uk^T q), scores and values come from the cache rows
//   expanded: the visible rows' keys and values per head are made first (W_uk c, W_uv c), for prompts
struct LatentShape {
    int heads, dim, rot, vdim, rank;
    int dp, rp, kp;              // dim rounded up to 8; rot and rank rounded up to 16
    float eps;
};
inline int latent_row(const LatentShape& s) { return s.kp + s.rp; }
inline int latent_q(const LatentShape& s) { return s.dp + s.rp; }

struct LatentCache {
    void* rows;                  // [sequence][max_seq][kp + rp]
    const int* past_len;
    int max_seq, seq;
    const float2* rope;          // [max_seq][rot / 2] cos, sin
};

// Raw projections -> rotated query rows and appended cache rows.
struct LatentFinish {
    LatentShape s;
    LatentCache cache;
    int f32;
    const float* q;              // [rows][ldq], a head's dp + rp columns at h (dp + rp); null: cache rows alone
    int ldq;
    const float* dkv;            // [rows][ld_dkv]: kp + rp columns; null: the rows belong to another layer
    int ld_dkv;
    const float* dkv_norm;       // [rank]
    void* q_out;                 // [rows][heads (dp + rp)], rotated
    void* q_abs;                 // [rows][heads (kp + rp)]: the rotated part (the rest is the absorbing product's), or null
};
int launch_latent_finish(const LatentFinish& p, int rows, cudaStream_t st);
// x / sqrt(mean(x^2) + eps) * norm over n columns, in the activation type, pads to ldo zero
int launch_rms_rows(const float* x, int ldx, int n, const float* norm, float eps, void* out, int ldo, int f32, int rows, cudaStream_t st);

struct LatentAttn {
    LatentShape s;
    LatentCache cache;
    int f32;
    const void* q_abs;           // [rows][heads (kp + rp)] in the activation type
    const float* q_raw;          // set: the rotated part is taken from here, [rows][ldq] raw
    int ldq;
    const float* dkv;            // set: the token's own cache row is made from here and appended (one token per sequence)
    int ld_dkv;
    const float* dkv_norm;
    int early;                   // earlier positions' cache rows may be read before the launch wait
    int window;
    float scale;
    const float* sinks;          // [heads], or null
    void* out;                   // [rows][heads kp]: weighted latents
};
bool latent_attn_supported(const LatentShape& s, int f32);
int launch_latent_attn(const LatentAttn& p, int rows, cudaStream_t st);

struct ExpandedAttn {
    LatentShape s;
    LatentCache cache;           // first sequence of this launch
    const __nv_bfloat16* q;      // [rows][heads (dp + rp)], rotated
    const __nv_bfloat16* kv;     // [sequence][len]: keys of every head (dp each), then values (vdim rounded up to 8 each)
    int first, len;              // cache positions first .. first + len - 1 are in kv
    int window;
    float scale;
    const float* sinks;
    const float* gate;           // [rows][ld_gate]: raw output gates, or null
    int ld_gate;
    __nv_bfloat16* out;          // [rows][ld_out]
    int ld_out;
};
bool expanded_attn_supported(const LatentShape& s, int seq);
int launch_expanded_attn(const ExpandedAttn& p, int batch, cudaStream_t st);

// Launch with programmatic dependent launch (kernels that wait before touching their predecessor's output).
template <typename... KArgs, typename... Args>
inline int launch_chained(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, int cluster,
                          Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    int n = 0;
    if (cluster > 1) {
        attr[n].id = cudaLaunchAttributeClusterDimension;
        attr[n].val.clusterDim.x = cluster;
        attr[n].val.clusterDim.y = 1;
        attr[n].val.clusterDim.z = 1;
        ++n;
    }
    if (g_use_pdl) {
        attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        attr[n].val.programmaticStreamSerializationAllowed = 1;
        ++n;
    }
    cfg.attrs = attr;
    cfg.numAttrs = n;
    if (cudaLaunchKernelEx(&cfg, kernel, args...) != cudaSuccess) {
        ++g_launch_count;
        cudaGetLastError();
        return ROTOR_B200_ERR_CUDA;
    }
    return launch_status();
}

#ifdef __CUDACC__
// Cached length of sequence b, kept inside the cache whatever the word holds.
__device__ __forceinline__ int cached_len(const int* past_len, int b, int max_seq) {
    return min(max(__ldg(past_len + b), 0), max_seq - 1);
}
// First position the query at `pos` sees.
__device__ __forceinline__ int first_visible(int pos, int chunk, int window) {
    const int c = chunk > 0 ? pos / chunk * chunk : 0, w = window > 0 ? pos - window + 1 : 0;
    return max(max(c, w), 0);
}
__device__ __forceinline__ float round_bf16(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }
__device__ __forceinline__ float4 bf16x4_to_float4(const uint2 u) {
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                       __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ uint2 float4_to_bf16x4(const float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    return make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
// 0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))) = z / (1 + exp(-2 sqrt(2/pi) (z + 0.044715 z^3)))
__device__ __forceinline__ float gelu_tanh(float z) {
    const float t = -1.5957691216057308f * (z + 0.044715f * z * z * z);
    return z / (1.0f + expf(fminf(t, 80.f)));
}

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gate_act(int act, float z) { return act == ACT_SILU ? silu(z) : gelu_tanh(z); }

// The `top` largest of a row's logits by one warp, the lower index first among equals: lane k < top gets the k-th
// expert and its softmax weight over the chosen ones.
__device__ __forceinline__ void route_row(const Routing& r, int row, int lane, int& sel, float& w) {
    const int experts = r.experts, top = r.top;
    auto logit = [&](int e) { return __ldcg(r.logits + (size_t)row * r.ld + e) + (r.bias ? __ldg(r.bias + e) : 0.f); };
    constexpr int KEPT = 4;  // logits per lane that stay in registers
    float kept[KEPT];
#pragma unroll
    for (int j = 0; j < KEPT; ++j) kept[j] = lane + 32 * j < experts ? logit(lane + 32 * j) : -INFINITY;
    // unsigned keys in the order of the values; what is not a number comes last
    auto key_of = [](float v) {
        const unsigned u = __float_as_uint(v);
        return v != v ? 0u : (u & 0x80000000u ? ~u : u | 0x80000000u);
    };
    unsigned last = 0xffffffffu;
    int last_i = -1;
    float mine = -INFINITY, first = 0.f;
    sel = 0;
    for (int k = 0; k < top; ++k) {
        unsigned best = 0u;
        int best_i = 0x7fffffff;
        float value = -INFINITY;
        auto offer = [&](int e, float v) {  // (in order of e)
            const unsigned q = key_of(v);
            if ((q < last || (q == last && e > last_i)) && (best_i == 0x7fffffff || q > best)) {
                best = q;
                best_i = e;
                value = v;
            }
        };
#pragma unroll
        for (int j = 0; j < KEPT; ++j)
            if (lane + 32 * j < experts) offer(lane + 32 * j, kept[j]);
        for (int e = lane + 32 * KEPT; e < experts; e += 32) offer(e, logit(e));
        const unsigned top_key = __reduce_max_sync(0xffffffffu, best);
        const int top_i = __reduce_min_sync(0xffffffffu, best == top_key ? best_i : 0x7fffffff);
        const float top_v = __shfl_sync(0xffffffffu, value, top_i & 31);  // (expert e is lane e % 32's)
        if (k == 0) first = top_v;
        if (lane == k) {
            sel = min(top_i, experts - 1);
            mine = top_v;
        }
        last = top_key;
        last_i = top_i;
    }
    const float e = lane < top ? expf(mine - first) : 0.f;
    w = e / warp_sum(e);
}

// Four columns (group g) of a stage's row, in two steps so that a thread can request several groups before
// it uses the first: the loads, then the new streams and their part of u.  `coef` (shared memory):
// mix [streams][streams], out [streams], in [streams].  S = 0: any number of streams (old streams are loaded
// in the second step).
template <int S>
struct StreamGroup {
    float4 y, x[S ? S : 1];  // (a first stage keeps the embedding's columns in y)
    // slot, slot_w: the row's part of slot_of and slot_w, wherever it lies (SLOTS: there may be any)
    template <bool SLOTS>
    __device__ __forceinline__ void load(const StreamStage& p, int row, int g, const int* slot, const float* slot_w) {
        if (p.ids) {
            long long id = p.ids[row];
            if (id < 0 || id >= p.vocab) id = 0;
            y = bf16x4_to_float4(__ldg(reinterpret_cast<const uint2*>(p.embed + (size_t)id * p.ld) + g));
            y = make_float4(y.x * p.embed_scale, y.y * p.embed_scale, y.z * p.embed_scale, y.w * p.embed_scale);
            return;
        }
        y = p.y ? __ldcg(reinterpret_cast<const float4*>(p.y + (size_t)row * p.ld) + g) : make_float4(0.f, 0.f, 0.f, 0.f);
        auto add = [&](const float4 v, float w) {
            y.x += w * v.x;
            y.y += w * v.y;
            y.z += w * v.z;
            y.w += w * v.w;
        };
        if (S <= 1 && p.y2) add(__ldcg(reinterpret_cast<const float4*>(p.y2 + (size_t)row * p.ld) + g), 1.f);
        if (SLOTS && p.slots && p.slots_f32) {
            for (int k = 0; k < p.top; ++k)
                add(__ldcg(reinterpret_cast<const float4*>(static_cast<const float*>(p.slots) + (size_t)slot[k] * p.ld) + g), slot_w[k]);
        } else if (SLOTS && p.slots) {
            constexpr int U = 4;  // slots requested together
            for (int k0 = 0; k0 < p.top; k0 += U) {
                uint2 v[U];
#pragma unroll
                for (int u = 0; u < U; ++u)
                    if (k0 + u < p.top)
                        v[u] = __ldcg(reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p.slots) + (size_t)slot[k0 + u] * p.ld) + g);
#pragma unroll
                for (int u = 0; u < U; ++u)
                    if (k0 + u < p.top) add(bf16x4_to_float4(v[u]), slot_w[k0 + u]);
            }
        }
        if constexpr (S > 0) {
            const float* xr = p.x_in + (size_t)row * S * p.ld;
#pragma unroll
            for (int s = 0; s < S; ++s) x[s] = __ldcg(reinterpret_cast<const float4*>(xr + (size_t)s * p.ld) + g);
        }
    }
    __device__ __forceinline__ float4 finish(const StreamStage& p, const float* coef, int row, int g, bool write) const {
        const int ns = S ? S : p.streams;
        const float* mix = coef;
        const float* out = coef + ns * ns;
        const float* in = out + ns;
        float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int t = 0; t < ns; ++t) {
            float4 v = y;
            if (!p.ids) {
                const float o = out[t];
                v = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
                for (int s = 0; s < ns; ++s) {
                    const float m = mix[s * ns + t];
                    float4 xs;
                    if constexpr (S > 0)
                        xs = x[s];
                    else
                        xs = __ldcg(reinterpret_cast<const float4*>(p.x_in + ((size_t)row * ns + s) * p.ld) + g);
                    v.x += m * xs.x;
                    v.y += m * xs.y;
                    v.z += m * xs.z;
                    v.w += m * xs.w;
                }
            }
            if (write) reinterpret_cast<float4*>(p.x_out + ((size_t)row * ns + t) * p.ld)[g] = v;
            const float i = in[t];
            u.x += i * v.x;
            u.y += i * v.y;
            u.z += i * v.z;
            u.w += i * v.w;
        }
        return u;
    }
};

// Four columns (group g) of a normed row; mean 0 and b null: root mean square norm.
__device__ __forceinline__ float4 norm_group(const float4 u, float mean, float inv, const float4 w, const float* b, int g) {
    float4 v = make_float4((u.x - mean) * inv * w.x, (u.y - mean) * inv * w.y, (u.z - mean) * inv * w.z, (u.w - mean) * inv * w.w);
    if (b) {
        const float4 c = __ldg(reinterpret_cast<const float4*>(b) + g);
        v = make_float4(v.x + c.x, v.y + c.y, v.z + c.z, v.w + c.w);
    }
    return v;
}
__device__ __forceinline__ float4 norm_group(const float4 u, float mean, float inv, const float* w, const float* b, int g) {
    return norm_group(u, mean, inv, __ldg(reinterpret_cast<const float4*>(w) + g), b, g);
}
// Sum of the squared deviations of a group's columns below n.
__device__ __forceinline__ float squared_deviations(const float4 u, float mean, int g, int n) {
    const float f[4] = {u.x, u.y, u.z, u.w};
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e)
        if (4 * g + e < n) ss += (f[e] - mean) * (f[e] - mean);
    return ss;
}

// The stage's coefficients into shared memory (they are weights: may run before the launch wait).
__device__ __forceinline__ void stream_coefs(const StreamStage& p, float* coef) {
    const int ns = p.streams;
    for (int i = threadIdx.x; i < ns * ns + 2 * ns; i += blockDim.x) {
        float v = 1.f;
        if (i < ns * ns)
            v = p.mix ? p.mix[i] : (ns == 1 ? 1.f : 0.f);
        else if (i < ns * ns + ns)
            v = p.out ? p.out[i - ns * ns] : (ns == 1 ? 1.f : 0.f);
        else if (p.in)
            v = p.in[i - ns * ns - ns];
        coef[i] = v;
    }
}
#endif

}  // namespace rb

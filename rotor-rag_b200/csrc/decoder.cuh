// Kernels of layer-described decoders: dense bf16 weights, residual streams with hyper-connections,
// attention with normalised queries and keys, a distance bias and a chunk mask, gated feed-forward.
// Every size and constant is a parameter; a design is a choice of them (decoder.cu).
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
// One stream with mix = in = out = 1 is the ordinary pre-norm residual.
struct StreamStage {
    int streams, n, ld;          // width and row stride of one stream
    const long long* ids;        // set: X_s <- embed[id] for every s instead of the mix
    const __nv_bfloat16* embed;  // [vocab][ld]
    int vocab;
    const float* x_in;           // [rows][streams][ld]
    float* x_out;                // [rows][streams][ld], not x_in; null: the new streams are not kept
    const float* y;              // [rows][ld]
    const float* mix;            // [from][to]
    const float* out;
    const float* in;
    const float* norm;           // [ld]
    float eps;
    const int* row_map;          // optional: output row r comes from source row row_map[r]
    void* h;                     // [rows][ldh]; columns past n are written as zeros
    int ldh;
    int h_f32;
};
int launch_stream_stage(const StreamStage& p, int rows, cudaStream_t st);

enum DenseEpilogue { DENSE_PLAIN = 0, DENSE_GATED = 1, DENSE_QKV = 2 };

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

// y[r][o] = sum_k x[r][k] w[o][k]
struct DenseProduct {
    const __nv_bfloat16* w;      // [n][ldw]; gated: [2 n][ldw], gate rows then up rows
    int n, k, ldw;
    int f32;                     // activation type
    const void* x;               // [rows][ldx]
    int ldx;
    const StreamStage* stage;    // few rows only: x is this stage's output, computed on the way
    int epilogue;                // DENSE_PLAIN: y float32; DENSE_GATED: a = gelu_tanh(gate) * up in the activation type
    float* y;
    int ldy;
    void* a;
    int lda;
    // DENSE_QKV (bf16): rows are [q heads | k heads | v heads]; normalised q rows out, k and v rows appended
    HeadShape shape;
    CacheView cache;
    __nv_bfloat16* q;            // [rows][heads * kd]
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

// softmax over the visible keys j of  (q . k_j) scale - slope (i - j);  j <= i, and j in i's chunk if chunk > 0
struct BiasAttn {
    HeadShape s;
    const float* qkv;            // raw projections: queries are normalised on the way (row kernel)
    int ld_qkv, f32;
    const __nv_bfloat16* q;      // normalised queries (tensor-core kernel)
    CacheView cache;
    int append;                  // one token per sequence: its key and value are taken from qkv and appended here
    int chunk;
    float scale;
    const float* slopes;         // [heads], or null for no bias
    void* out;                   // [rows][ld_out], head h at column h * vdim
    int ld_out;
};
int bias_attn_reach(const BiasAttn& p);  // most keys one query can see
int launch_bias_attn_rows(const BiasAttn& p, int rows, cudaStream_t st);
bool bias_attn_t5_supported(const BiasAttn& p, int rows);
int launch_bias_attn_t5(const BiasAttn& p, int rows, cudaStream_t st);

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

// Four columns (group g) of a stage's row, in two steps so that a thread can request several groups before
// it uses the first: the loads, then the new streams and their part of u.  `coef` (shared memory):
// mix [streams][streams], out [streams], in [streams].  S = 0: any number of streams (old streams are loaded
// in the second step).
template <int S>
struct StreamGroup {
    float4 y, x[S ? S : 1];  // (a first stage keeps the embedding's columns in y)
    __device__ __forceinline__ void load(const StreamStage& p, int row, int g) {
        if (p.ids) {
            long long id = p.ids[row];
            if (id < 0 || id >= p.vocab) id = 0;
            y = bf16x4_to_float4(__ldg(reinterpret_cast<const uint2*>(p.embed + (size_t)id * p.ld) + g));
            return;
        }
        y = __ldcg(reinterpret_cast<const float4*>(p.y + (size_t)row * p.ld) + g);
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

// The stage's coefficients into shared memory (they are weights: may run before the launch wait).
__device__ __forceinline__ void stream_coefs(const StreamStage& p, float* coef) {
    const int ns = p.streams;
    for (int i = threadIdx.x; i < ns * ns + 2 * ns; i += blockDim.x) {
        float v = 1.f;
        if (i < ns * ns)
            v = p.mix ? p.mix[i] : 0.f;
        else if (i < ns * ns + ns)
            v = p.out ? p.out[i - ns * ns] : 0.f;
        else if (p.in)
            v = p.in[i - ns * ns - ns];
        coef[i] = v;
    }
}
#endif

}  // namespace rb

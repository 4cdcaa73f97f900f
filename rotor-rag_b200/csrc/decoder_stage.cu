// Row-wise stages of layer-described decoders: residual streams with hyper-connections and the
// norms that follow (stream_stage_kernel), and the split of projection rows into normalised queries and
// appended cache rows (head_finish_kernel).
#include "decoder.cuh"

namespace rb {

// One row per CTA pass; u stays in shared memory between the sum of squares and the scaling.
template <int S>
__global__ void __launch_bounds__(256) stream_stage_kernel(const __grid_constant__ StreamStage p, int rows) {
    extern __shared__ __align__(16) float us[];  // [ld]
    __shared__ float coef[STREAMS_MAX * STREAMS_MAX + 2 * STREAMS_MAX], red[64], slot_w[EXPERT_TOP_MAX];
    __shared__ int slot[EXPERT_TOP_MAX];
    stream_coefs(p, coef);
    pdl_wait();
    pdl_trigger();
    __syncthreads();
    const int n4 = p.ld >> 2;
    int k = 0;
    for (int r = blockIdx.x; r < rows; r += gridDim.x) {
        const int src = p.row_map ? p.row_map[r] : r;
        if (p.slots) {
            __syncthreads();  // (the row before is done with them)
            if ((int)threadIdx.x < p.top) {
                slot[threadIdx.x] = __ldcg(p.slot_of + (size_t)src * p.top + threadIdx.x);
                slot_w[threadIdx.x] = __ldcg(p.slot_w + (size_t)src * p.top + threadIdx.x);
            }
            __syncthreads();
        }
        float ss = 0.f;
        constexpr int U = S == 1 ? 2 : 1;  // groups per thread requested together
        for (int g0 = threadIdx.x; g0 < n4; g0 += U * blockDim.x) {
            StreamGroup<S> sg[U];
#pragma unroll
            for (int i = 0; i < U; ++i)
                if (g0 + i * (int)blockDim.x < n4) sg[i].template load<true>(p, src, g0 + i * blockDim.x, slot, slot_w);
#pragma unroll
            for (int i = 0; i < U; ++i) {
                const int g = g0 + i * blockDim.x;
                if (g >= n4) break;
                const float4 u = sg[i].finish(p, coef, src, g, p.x_out != nullptr);
                ss += p.norm_b ? u.x + u.y + u.z + u.w : u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
                reinterpret_cast<float4*>(us)[g] = u;
            }
        }
        if (!p.h) continue;
        float mean = 0.f;
        ss = block_sum_alt(ss, red, k);
        if (p.norm_b) {  // own groups of us
            mean = ss / (float)p.n;
            ss = 0.f;
            for (int g = threadIdx.x; g < n4; g += blockDim.x) ss += squared_deviations(reinterpret_cast<const float4*>(us)[g], mean, g, p.n);
            ss = block_sum_alt(ss, red, k);
        }
        const float inv = 1.0f / sqrtf(ss / (float)p.n + p.eps);
        auto store = [&](void* h, int g, const float4 v) {
            if (p.h_f32)
                reinterpret_cast<float4*>(static_cast<float*>(h) + (size_t)r * p.ldh)[g] = v;
            else
                reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(h) + (size_t)r * p.ldh)[g] = float4_to_bf16x4(v);
        };
        for (int g = threadIdx.x; g < (p.ldh >> 2); g += blockDim.x) {  // own groups of us, zeros behind them
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f), u = v;
            if (g < n4) {
                u = reinterpret_cast<const float4*>(us)[g];
                v = norm_group(u, mean, inv, p.norm, p.norm_b, g);
            }
            store(p.h, g, v);
            if (p.norm2) store(p.h2, g, g < n4 ? norm_group(u, mean, inv, p.norm2, p.norm2_b, g) : v);
        }
    }
}

int launch_stream_stage(const StreamStage& p, int rows, cudaStream_t st) {
    RB_REQUIRE(rows > 0 && p.streams >= 1 && p.streams <= STREAMS_MAX && p.ld % 4 == 0 && p.ldh % 4 == 0);
    const size_t smem = (size_t)p.ld * sizeof(float);
    if (smem > 40 * 1024) return ROTOR_B200_ERR_SHAPE;
    RB_REQUIRE(!p.norm2 || (p.h && p.h2 && (p.norm_b != nullptr) == (p.norm2_b != nullptr)));
    const int threads = p.ld >= 1024 ? 256 : (p.ld >= 256 ? 128 : 64);
    const int per_sm = 2048 / threads;
    dim3 grid(rows < 148 * per_sm ? rows : 148 * per_sm), block(threads);
    switch (p.streams) {
        case 1: return launch_chained(stream_stage_kernel<1>, grid, block, smem, st, 1, p, rows);
        case 2: return launch_chained(stream_stage_kernel<2>, grid, block, smem, st, 1, p, rows);
        case 3: return launch_chained(stream_stage_kernel<3>, grid, block, smem, st, 1, p, rows);
        case 4: return launch_chained(stream_stage_kernel<4>, grid, block, smem, st, 1, p, rows);
        default: return launch_chained(stream_stage_kernel<0>, grid, block, smem, st, 1, p, rows);
    }
}

// One warp per head vector of a row.
__global__ void __launch_bounds__(256) head_finish_kernel(const __grid_constant__ HeadFinish p, int rows) {
    const HeadShape& s = p.s;
    const int lane = threadIdx.x & 31;
    const int vecs = s.heads + 2 * s.kv_heads, first = p.q ? 0 : s.heads;
    const int per = vecs - first;
    const long long total = (long long)rows * per;
    const long long nw = (long long)gridDim.x * (blockDim.x >> 5);
    for (long long i = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5); i < total; i += nw) {
        const int row = (int)(i / per), v = first + (int)(i - (long long)row * per);
        const bool is_v = v >= s.heads + s.kv_heads;
        const int len = is_v ? s.vdim : s.dim, wide = is_v ? s.vd : s.kd;
        const float* src = p.qkv + (size_t)row * p.ld_qkv +
                           (is_v ? (s.heads + s.kv_heads) * s.dim + (v - s.heads - s.kv_heads) * s.vdim : v * s.dim);
        float inv = 1.f;
        if (s.unit && !is_v) {
            float ss = 0.f;
            for (int c = lane; c < len; c += 32) ss += src[c] * src[c];
            inv = 1.0f / sqrtf(warp_sum(ss) / (float)len + s.eps);
        }
        size_t dst;  // element offset of the output row
        if (v < s.heads) {
            dst = ((size_t)row * s.heads + v) * s.kd;
        } else {
            const int b = row / p.cache.seq, pos = cached_len(p.cache.past_len, b, p.cache.max_seq) + (row - b * p.cache.seq);
            const int head = is_v ? v - s.heads - s.kv_heads : v - s.heads;
            if (pos >= p.cache.max_seq) continue;
            dst = (((size_t)b * s.kv_heads + head) * p.cache.max_seq + pos) * wide;
        }
        for (int c = lane; c < wide; c += 32) {
            const float x = c < len ? src[c] * inv : 0.f;
            if (v < s.heads)
                p.q[dst + c] = __float2bfloat16_rn(x);
            else if (p.f32)
                static_cast<float*>(is_v ? p.cache.v : p.cache.k)[dst + c] = x;
            else
                static_cast<__nv_bfloat16*>(is_v ? p.cache.v : p.cache.k)[dst + c] = __float2bfloat16_rn(x);
        }
    }
}

int launch_head_finish(const HeadFinish& p, int rows, cudaStream_t st) {
    const long long total = (long long)rows * (p.s.heads + 2 * p.s.kv_heads);
    const long long blocks = (total + 7) / 8;
    head_finish_kernel<<<(unsigned)(blocks < 148 * 8 ? blocks : 148 * 8), 256, 0, st>>>(p, rows);
    return launch_status();
}

}  // namespace rb

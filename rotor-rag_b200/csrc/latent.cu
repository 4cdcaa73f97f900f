// Latent attention in the latent space (the absorbed form), one query position at a time:
//   score_h(i, j) = (W_uk,h^T q_i,h . c_j + rot(q_i,h) . rot(k_j)) scale,   j <= i, and i - j < window
//   out_h(i)      = sum_j p_h(i, j) c_j,   the softmax's denominator holding exp(sink_h) as well
// where a cached position is one row [c | rot(k)] for all heads, read once as key and as value.  Used by
// generation steps (the new row is normed, rotated and appended here), short portions and float32 runs;
// prompts go through attn_bias_t5.cu in the expanded form.
//
// Grid (splits, head tiles, rows); the splits of a row form a thread-block cluster.  A CTA takes an equal run of
// the row's visible positions for one tile of heads, walks it in tiles of cache rows staged by cp.async (the
// first requested before the programmatic-launch wait where it holds only rows of earlier steps), keeps a
// running maximum and sum per head, and the cluster merges through distributed shared memory.
//   bf16:    16 heads a tile are the M of mma.m16n8k16: warps split the positions and halves of a row for the
//            scores and the latent columns for the sums
//   float32: the FP32 pipe, eight heads a tile
#include "decoder.cuh"

namespace rb {

constexpr int LA_THREADS = 512, LA_WARPS = LA_THREADS / 32;
constexpr int LA_HEADS = 16, LF_HEADS = 8;
constexpr int LA_MAX_SPLITS = 16;           // (above eight: clusters of a size the device has to allow)
constexpr size_t LA_SMEM_MAX = 200 * 1024;

struct LatentArgs {
    LatentAttn p;
    int row0, tile;
};

// ---------------------------------------------------------------- row-wise pieces
__device__ __forceinline__ float2 rot_pair(const float2 v, const float2 cs) { return make_float2(v.x * cs.x - v.y * cs.y, v.y * cs.x + v.x * cs.y); }
__device__ __forceinline__ void la_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void la_store(float* p, float v) { *p = v; }
__device__ __forceinline__ void la_store2(__nv_bfloat16* p, const float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }
__device__ __forceinline__ void la_store2(float* p, const float2 v) { *reinterpret_cast<float2*>(p) = v; }

// One warp makes a cache row from its raw projection: put(column, value pair) for all kp + rp columns.
template <typename F>
__device__ __forceinline__ void latent_cache_row(const LatentShape& s, const float* raw, const float* norm, const float2* rope, int lane, F put) {
    constexpr int U = 8;  // column pairs per lane that stay in registers
    float2 keep[U];
    float ss = 0.f;
    auto pair = [&](int c) {  // (the columns between rank and kp are zeros)
        return 2 * c < s.kp ? __ldcg(reinterpret_cast<const float2*>(raw) + c) : make_float2(0.f, 0.f);
    };
#pragma unroll
    for (int u = 0; u < U; ++u) keep[u] = pair(lane + 32 * u);
#pragma unroll
    for (int u = 0; u < U; ++u) ss += keep[u].x * keep[u].x + keep[u].y * keep[u].y;
    for (int c = lane + 32 * U; 2 * c < s.kp; c += 32) {
        const float2 v = pair(c);
        ss += v.x * v.x + v.y * v.y;
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)s.rank + s.eps);
    auto scaled = [&](int c, const float2 v) {
        if (2 * c < s.kp)
            put(2 * c, make_float2(2 * c < s.rank ? v.x * inv * __ldg(norm + 2 * c) : 0.f, 2 * c + 1 < s.rank ? v.y * inv * __ldg(norm + 2 * c + 1) : 0.f));
    };
#pragma unroll
    for (int u = 0; u < U; ++u) scaled(lane + 32 * u, keep[u]);
    for (int c = lane + 32 * U; 2 * c < s.kp; c += 32) scaled(c, pair(c));
    for (int i = lane; i < (s.rp >> 1); i += 32) {
        const float2 v = __ldcg(reinterpret_cast<const float2*>(raw + s.kp) + i);
        put(s.kp + 2 * i, 2 * i < s.rot ? rot_pair(v, __ldg(rope + i)) : make_float2(0.f, 0.f));
    }
}

// One warp per query head and, behind them, per cache row.
template <typename T>
__global__ void __launch_bounds__(256) latent_finish_kernel(const __grid_constant__ LatentFinish p, int rows) {
    pdl_wait();
    pdl_trigger();
    const LatentShape& s = p.s;
    const int lane = threadIdx.x & 31, W = s.kp + s.rp, qd = s.dp + s.rp;
    const int per = (p.q ? s.heads : 0) + (p.dkv ? 1 : 0);
    const long long total = (long long)rows * per, nw = (long long)gridDim.x * (blockDim.x >> 5);
    for (long long i = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5); i < total; i += nw) {
        const int row = (int)(i / per), v = (int)(i - (long long)row * per);
        const int b = row / p.cache.seq, pos = cached_len(p.cache.past_len, b, p.cache.max_seq) + (row - b * p.cache.seq);
        if (pos >= p.cache.max_seq) continue;
        const float2* rope = p.cache.rope + (size_t)pos * (s.rot >> 1);
        if (p.q && v < s.heads) {
            const float2* src = reinterpret_cast<const float2*>(p.q + (size_t)row * p.ldq + (size_t)v * qd);
            T* dst = static_cast<T*>(p.q_out) + ((size_t)row * s.heads + v) * qd;
            for (int c = lane; c < (qd >> 1); c += 32) {
                float2 x = src[c];
                const int r = c - (s.dp >> 1);
                if (r >= 0) {
                    x = 2 * r < s.rot ? rot_pair(x, __ldg(rope + r)) : make_float2(0.f, 0.f);
                    if (p.q_abs) la_store2(static_cast<T*>(p.q_abs) + ((size_t)row * s.heads + v) * W + s.kp + 2 * r, x);
                }
                la_store2(dst + 2 * c, x);
            }
        } else {
            T* dst = static_cast<T*>(p.cache.rows) + ((size_t)b * p.cache.max_seq + pos) * W;
            latent_cache_row(s, p.dkv + (size_t)row * p.ld_dkv, p.dkv_norm, rope, lane, [&](int c, const float2 x) { la_store2(dst + c, x); });
        }
    }
}

int launch_latent_finish(const LatentFinish& p, int rows, cudaStream_t st) {
    const int per = (p.q ? p.s.heads : 0) + (p.dkv ? 1 : 0);
    if (!per) return ROTOR_B200_OK;
    RB_REQUIRE(rows > 0 && p.cache.rows && p.cache.past_len && p.cache.rope && (!p.q || p.q_out) && (!p.dkv || p.dkv_norm));
    RB_REQUIRE(p.ldq % 2 == 0 && p.ld_dkv % 2 == 0);
    const long long blocks = ((long long)rows * per + 7) / 8;
    const dim3 grid((unsigned)(blocks < 148 * 8 ? blocks : 148 * 8));
    return p.f32 ? launch_chained(latent_finish_kernel<float>, grid, dim3(256), 0, st, 1, p, rows)
                 : launch_chained(latent_finish_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, 1, p, rows);
}

// One CTA per row.
template <typename T>
__global__ void __launch_bounds__(256) rms_rows_kernel(const float* x, int ldx, int n, const float* norm, float eps, T* out, int ldo, int rows) {
    __shared__ float red[64];
    pdl_wait();
    pdl_trigger();
    int k = 0;
    for (int r = blockIdx.x; r < rows; r += gridDim.x) {
        const float2* v = reinterpret_cast<const float2*>(x + (size_t)r * ldx);
        constexpr int U = 4;  // column pairs per thread that stay in registers
        float2 keep[U];
        float ss = 0.f;
        auto pair = [&](int c) {
            float2 q = 2 * c < n ? v[c] : make_float2(0.f, 0.f);
            if (2 * c + 1 >= n) q.y = 0.f;
            ss += q.x * q.x + q.y * q.y;
            return q;
        };
#pragma unroll
        for (int u = 0; u < U; ++u) keep[u] = pair(threadIdx.x + u * blockDim.x);
        for (int c = threadIdx.x + U * blockDim.x; 2 * c < n; c += blockDim.x) pair(c);
        const float inv = 1.0f / sqrtf(block_sum_alt(ss, red, k) / (float)n + eps);
        auto put = [&](int c, const float2 q) {
            if (2 * c < ldo)
                la_store2(out + (size_t)r * ldo + 2 * c, make_float2(2 * c < n ? q.x * inv * __ldg(norm + 2 * c) : 0.f,
                                                                     2 * c + 1 < n ? q.y * inv * __ldg(norm + 2 * c + 1) : 0.f));
        };
#pragma unroll
        for (int u = 0; u < U; ++u) put(threadIdx.x + u * blockDim.x, keep[u]);
        for (int c = threadIdx.x + U * blockDim.x; 2 * c < ldo; c += blockDim.x) put(c, pair(c));
    }
}

int launch_rms_rows(const float* x, int ldx, int n, const float* norm, float eps, void* out, int ldo, int f32, int rows, cudaStream_t st) {
    RB_REQUIRE(x && norm && out && rows > 0 && n > 0 && n <= ldo && ldx % 2 == 0 && ldo % 2 == 0);
    const dim3 grid(rows < 148 * 8 ? rows : 148 * 8);
    return f32 ? launch_chained(rms_rows_kernel<float>, grid, dim3(256), 0, st, 1, x, ldx, n, norm, eps, static_cast<float*>(out), ldo, rows)
               : launch_chained(rms_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, 1, x, ldx, n, norm, eps,
                                static_cast<__nv_bfloat16*>(out), ldo, rows);
}

// ---------------------------------------------------------------- attention
__device__ __forceinline__ uint32_t la_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ float la_ld_cluster(const float* local, unsigned rank) {
    uint32_t a;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(la_smem(local)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
    return v;
}
__device__ __forceinline__ void la_cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

// The run of one CTA, and the loads of its tiles.
template <typename T>
struct LatentRun {
    static constexpr int PIECE = 16 / (int)sizeof(T);
    int row, pos, t0, t1, W, stride;
    T* rows;
    __device__ LatentRun(const LatentArgs& a, int rank, int ns) {
        const LatentAttn& p = a.p;
        W = p.s.kp + p.s.rp;
        stride = W + PIECE;  // staged rows start an odd number of 16-byte pieces apart: column reads without bank conflicts
        row = a.row0 + (int)blockIdx.z;
        const int b = row / p.cache.seq;
        pos = min(cached_len(p.cache.past_len, b, p.cache.max_seq) + (row - b * p.cache.seq), p.cache.max_seq - 1);
        const int lo = first_visible(pos, 0, p.window), per = (pos + 1 - lo + ns - 1) / ns;
        t0 = lo + rank * per;
        t1 = min(t0 + per, pos + 1);
        rows = static_cast<T*>(p.cache.rows) + (size_t)b * p.cache.max_seq * W;
    }
    // cache rows k0 .. k0 + tile - 1 below t1, `skip` left out; rows behind them as zeros
    __device__ __forceinline__ void load(T* dst, int k0, int tile, int skip) const {
        const int n = min(tile, t1 - k0), pieces = W / PIECE;
        for (int j = threadIdx.x >> 5; j < tile; j += LA_WARPS) {
            if (k0 + j == skip && j < n) continue;
            const int bytes = j < n ? 16 : 0;
            const T* src = rows + (size_t)(j < n ? k0 + j : k0) * W;
            const uint32_t to = la_smem(dst + (size_t)j * stride);
            for (int c = threadIdx.x & 31; c < pieces; c += 32)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(to + 16 * c), "l"(src + c * PIECE), "r"(bytes) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    }
};

// Merges the cluster's runs, every CTA a share of the outputs.  po: this CTA's un-normalised sums [heads][stride],
// ml: maxima (base-2 exponents) [hb], sums at ml + hb.
template <typename T>
__device__ __forceinline__ void la_merge(const LatentAttn& p, const float* po, int stride, const float* ml, int hb, int h0, int nh, int row, int rank,
                                         int ns) {
    if (ns > 1)
        la_cluster_sync();
    else
        __syncthreads();
    const int kp = p.s.kp;
    T* out = static_cast<T*>(p.out) + ((size_t)row * p.s.heads + h0) * kp;
    for (int idx = rank * LA_THREADS + (int)threadIdx.x; idx < nh * (kp >> 1); idx += ns * LA_THREADS) {
        const int h = idx / (kp >> 1), c = (idx - h * (kp >> 1)) * 2;
        const float sink = p.sinks ? __ldg(p.sinks + h0 + h) * 1.4426950408889634f : -INFINITY;
        float2 o;
        float l, M = sink;
        if (ns == 1) {
            M = fmaxf(M, ml[h]);
            const float e = exp2f(ml[h] - M);
            o = make_float2(e * po[h * stride + c], e * po[h * stride + c + 1]);
            l = e * ml[hb + h];
        } else {
            float m[LA_MAX_SPLITS], w[LA_MAX_SPLITS];
            float2 v[LA_MAX_SPLITS];
#pragma unroll
            for (int k = 0; k < LA_MAX_SPLITS; ++k) {  // (all remote reads in flight together)
                m[k] = k < ns ? la_ld_cluster(ml + h, k) : -INFINITY;
                w[k] = k < ns ? la_ld_cluster(ml + hb + h, k) : 0.f;
                v[k].x = k < ns ? la_ld_cluster(po + h * stride + c, k) : 0.f;
                v[k].y = k < ns ? la_ld_cluster(po + h * stride + c + 1, k) : 0.f;
            }
#pragma unroll
            for (int k = 0; k < LA_MAX_SPLITS; ++k) M = fmaxf(M, m[k]);
            o = make_float2(0.f, 0.f);
            l = 0.f;
#pragma unroll
            for (int k = 0; k < LA_MAX_SPLITS; ++k) {
                const float e = exp2f(m[k] - M);
                l += e * w[k];
                o.x += e * v[k].x;
                o.y += e * v[k].y;
            }
        }
        l += exp2f(sink - M);
        la_store2(out + (size_t)h * kp + c, make_float2(o.x / l, o.y / l));
    }
    if (ns > 1) la_cluster_sync();  // nobody leaves while its shared memory may still be read
}

// The query rows of a CTA's heads into shared memory (rows of `stride`); rows past nh are zeros.
template <typename T>
__device__ __forceinline__ void la_queries(const LatentAttn& p, T* qs, int stride, int h0, int nh, int tile_heads, int row, const float2* rope) {
    const LatentShape& s = p.s;
    constexpr int PIECE = 16 / (int)sizeof(T), U = 3;  // pieces per thread requested together
    const int W = s.kp + s.rp, from = p.q_raw ? s.kp : W, pieces = from / PIECE, total = tile_heads * pieces;
    const T* q = static_cast<const T*>(p.q_abs) + ((size_t)row * s.heads + h0) * W;
    // the rotated part from the raw projections: requested first, turned last
    const int pairs = p.q_raw ? s.rp >> 1 : 0, rots = tile_heads * pairs;
    float2 raw = make_float2(0.f, 0.f), cs = raw;
    auto rot_of = [&](int i, float2& x, float2& t) {
        const int h = i / pairs, r = i - h * pairs;
        x = t = make_float2(0.f, 0.f);
        if (h < nh && 2 * r < s.rot) {
            x = __ldcg(reinterpret_cast<const float2*>(p.q_raw + (size_t)row * p.ldq + (size_t)(h0 + h) * (s.dp + s.rp) + s.dp) + r);
            t = __ldg(rope + r);
        }
    };
    if ((int)threadIdx.x < rots) rot_of(threadIdx.x, raw, cs);
    for (int i0 = threadIdx.x; i0 < total; i0 += U * LA_THREADS) {
        uint4 v[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int i = i0 + u * LA_THREADS, h = i / pieces, c = i - h * pieces;
            v[u] = make_uint4(0u, 0u, 0u, 0u);
            if (i < total && h < nh) v[u] = __ldcg(reinterpret_cast<const uint4*>(q + (size_t)h * W) + c);
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int i = i0 + u * LA_THREADS, h = i / pieces, c = i - h * pieces;
            if (i < total) *reinterpret_cast<uint4*>(qs + h * stride + c * PIECE) = v[u];
        }
    }
    for (int i = threadIdx.x; i < rots; i += LA_THREADS) {
        if (i != (int)threadIdx.x) rot_of(i, raw, cs);
        const int h = i / pairs, r = i - h * pairs;
        la_store2(qs + h * stride + s.kp + 2 * r, rot_pair(raw, cs));
    }
}

__device__ __forceinline__ void la_ldm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void la_ldm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void la_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// NC: blocks of 16 latent columns per warp.
template <int NC>
__global__ void __launch_bounds__(LA_THREADS) latent_attn_mma_kernel(const __grid_constant__ LatentArgs a) {
    typedef __nv_bfloat16 T;
    const LatentAttn& p = a.p;
    const LatentShape& s = p.s;
    extern __shared__ __align__(16) unsigned char la_raw[];
    const int ns = (int)gridDim.x, rank = (int)blockIdx.x, h0 = (int)blockIdx.y * LA_HEADS, nh = min(LA_HEADS, s.heads - h0);
    const LatentRun<T> run(a, rank, ns);
    const int TK = a.tile, W = run.W, ws = run.stride, ss = TK + 4, ps_ld = TK + 8;
    T* qs = reinterpret_cast<T*>(la_raw);                        // [16][ws]
    T* kv = qs + LA_HEADS * ws;                                  // [2][TK][ws]; at the end the CTA's sums, float [16][kp + 4]
    T* ps = kv + 2 * (size_t)TK * ws;                            // [16][TK + 8] weights
    float* sc = reinterpret_cast<float*>(ps + LA_HEADS * ps_ld); // [2][16][TK + 4] scores, by halves of the row
    float* ml = sc + 2 * LA_HEADS * ss;                             // m [16], l [16], alpha [16]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const float2* rope = p.cache.rope + (size_t)run.pos * (s.rot >> 1);
    const int skip = p.dkv ? run.pos : -1;

    if (p.early && run.t0 < run.t1) run.load(kv, run.t0, TK, skip);
    if (p.dkv && warp == 0) {  // constants the new row needs
        for (int c = lane * 32; c < s.rank; c += 32 * 32) prefetch_l2(p.dkv_norm + c);
        if (lane * 16 < (s.rot >> 1)) prefetch_l2(rope + lane * 16);
    }
    pdl_wait();
    pdl_trigger();
    if (!p.early && run.t0 < run.t1) run.load(kv, run.t0, TK, skip);
    const bool owner = p.dkv && run.t0 <= run.pos && run.pos < run.t1;  // (the last position of the run)
    if (owner && warp == 0) {
        const int k0 = (run.pos - run.t0) / TK * TK + run.t0;
        T* stage = kv + (size_t)(((k0 - run.t0) / TK & 1) * TK + (run.pos - k0)) * ws;
        T* dst = run.rows + (size_t)run.pos * W;
        // straight into its tile if that is the first, else into the cache and from there by the copies of its tile
        latent_cache_row(s, p.dkv + (size_t)run.row * p.ld_dkv, p.dkv_norm, rope, lane, [&](int c, const float2 x) {
            if (k0 == run.t0) la_store2(stage + c, x);
            if (blockIdx.y == 0 || k0 != run.t0) la_store2(dst + c, x);
        });
        if (k0 != run.t0) __threadfence();
    }
    la_queries(p, qs, ws, h0, nh, LA_HEADS, run.row, rope);
    if (tid < LA_HEADS) {
        ml[tid] = -INFINITY;
        ml[LA_HEADS + tid] = 0.f;
    }

    float o[NC][2][4];
#pragma unroll
    for (int i = 0; i < NC; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[i][j][e] = 0.f;
    const float scale2 = p.scale * 1.4426950408889634f;
    const uint32_t qa = la_smem(qs + (size_t)(lane & 15) * ws + (lane >> 4) * 8);
    for (int k0 = run.t0, it = 0; k0 < run.t1; k0 += TK, ++it) {
        const T* tile = kv + (size_t)(it & 1) * TK * ws;
        const int n = min(TK, run.t1 - k0);
        __syncthreads();  // the other buffer's readers are done, and the new row (first tile or cache) is written
        if (k0 + TK < run.t1) {
            run.load(kv + (size_t)((it & 1) ^ 1) * TK * ws, k0 + TK, TK, -1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        // scores of eight positions per warp, over half of the row
        {
            const int kb = (warp & 7) * 8, part = warp >> 3, mid = (W / 16 + 1) / 2 * 16;
            if (kb < TK) {
                float d0[4] = {0.f, 0.f, 0.f, 0.f}, d1[4] = {0.f, 0.f, 0.f, 0.f};
                const uint32_t ka = la_smem(tile + (size_t)(kb + (lane & 7)) * ws + (lane >> 3) * 8);
                const int end = part ? W : mid;
                int c = part ? mid : 0;
#pragma unroll 3
                for (; c + 32 <= end; c += 32) {
                    uint32_t q0[4], q1[4], b[4];
                    la_ldm4(b, ka + c * 2);
                    la_ldm4(q0, qa + c * 2);
                    la_ldm4(q1, qa + c * 2 + 32);
                    la_mma(d0, q0, b[0], b[1]);
                    la_mma(d1, q1, b[2], b[3]);
                }
                if (c < end) {
                    uint32_t q0[4], b0, b1;
                    const uint32_t kt = la_smem(tile + (size_t)(kb + (lane & 7)) * ws + ((lane >> 3) & 1) * 8 + c);
                    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(b0), "=r"(b1) : "r"(kt));
                    la_ldm4(q0, qa + c * 2);
                    la_mma(d0, q0, b0, b1);
                }
                float* to = sc + (size_t)part * LA_HEADS * ss + (lane >> 2) * ss + kb + (lane & 3) * 2;
                *reinterpret_cast<float2*>(to) = make_float2(d0[0] + d1[0], d0[1] + d1[1]);
                *reinterpret_cast<float2*>(to + 8 * ss) = make_float2(d0[2] + d1[2], d0[3] + d1[3]);
            }
        }
        __syncthreads();
        static_assert(LA_HEADS == LA_WARPS, "a warp per head");
        {
            const int h = warp;
            float v[2], top = -INFINITY, sum = 0.f;  // (tiles of up to 64 positions)
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int k = lane + 32 * i;
                v[i] = k < n ? (sc[h * ss + k] + sc[(LA_HEADS + h) * ss + k]) * scale2 : -INFINITY;
                top = fmaxf(top, v[i]);
            }
            const float m_old = ml[h], m_new = fmaxf(m_old, warp_max(top));  // finite: a tile has a visible position
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int k = lane + 32 * i;
                v[i] = exp2f(v[i] - m_new);
                if (k < TK) ps[h * ps_ld + k] = __float2bfloat16_rn(v[i]);
                sum += v[i];
            }
            sum = warp_sum(sum);
            if (lane == 0) {
                const float al = exp2f(m_old - m_new);
                ml[h] = m_new;
                ml[LA_HEADS + h] = ml[LA_HEADS + h] * al + sum;
                ml[2 * LA_HEADS + h] = al;
            }
        }
        __syncthreads();
        const float al0 = ml[2 * LA_HEADS + (lane >> 2)], al1 = ml[2 * LA_HEADS + (lane >> 2) + 8];
#pragma unroll
        for (int i = 0; i < NC; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                o[i][j][0] *= al0;
                o[i][j][1] *= al0;
                o[i][j][2] *= al1;
                o[i][j][3] *= al1;
            }
        const uint32_t pa = la_smem(ps + (size_t)(lane & 15) * ps_ld + (lane >> 4) * 8);
        for (int kk = 0; kk < n; kk += 16) {
            uint32_t w[4];
            la_ldm4(w, pa + kk * 2);
            const uint32_t va = la_smem(tile + (size_t)(kk + (lane & 15)) * ws + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < NC; ++i) {
                const int cb = warp + i * LA_WARPS;
                if (cb * 16 < s.kp) {
                    uint32_t v[4];
                    la_ldm4t(v, va + cb * 32);
                    la_mma(o[i][0], w, v[0], v[1]);
                    la_mma(o[i][1], w, v[2], v[3]);
                }
            }
        }
    }
    __syncthreads();
    float* po = reinterpret_cast<float*>(kv);
    const int po_ld = s.kp + 4;
#pragma unroll
    for (int i = 0; i < NC; ++i) {
        const int cb = warp + i * LA_WARPS;
        if (cb * 16 < s.kp) {
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                float* d = po + (lane >> 2) * po_ld + cb * 16 + j * 8 + (lane & 3) * 2;
                *reinterpret_cast<float2*>(d) = make_float2(o[i][j][0], o[i][j][1]);
                *reinterpret_cast<float2*>(d + 8 * po_ld) = make_float2(o[i][j][2], o[i][j][3]);
            }
        }
    }
    la_merge<T>(p, po, po_ld, ml, LA_HEADS, h0, nh, run.row, rank, ns);
}

__global__ void __launch_bounds__(LA_THREADS) latent_attn_f32_kernel(const __grid_constant__ LatentArgs a) {
    const LatentAttn& p = a.p;
    const LatentShape& s = p.s;
    extern __shared__ __align__(16) unsigned char la_raw[];
    const int ns = (int)gridDim.x, rank = (int)blockIdx.x, h0 = (int)blockIdx.y * LF_HEADS, nh = min(LF_HEADS, s.heads - h0);
    const LatentRun<float> run(a, rank, ns);
    const int TK = a.tile, W = run.W, ws = run.stride, po_ld = s.kp + 4;
    float* qs = reinterpret_cast<float*>(la_raw);  // [8][ws]
    float* kv = qs + LF_HEADS * ws;                // [TK][ws]
    float* sc = kv + (size_t)TK * ws;              // [8][TK]
    float* po = sc + LF_HEADS * TK;                // [8][kp + 4]
    float* ml = po + LF_HEADS * po_ld;             // m, l, alpha [8]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const float2* rope = p.cache.rope + (size_t)run.pos * (s.rot >> 1);
    pdl_wait();
    pdl_trigger();
    la_queries(p, qs, ws, h0, nh, LF_HEADS, run.row, rope);
    const bool owner = p.dkv && run.t0 <= run.pos && run.pos < run.t1;
    if (owner && warp == 0) {
        float* dst = run.rows + (size_t)run.pos * W;  // (every tile of heads writes the same values)
        latent_cache_row(s, p.dkv + (size_t)run.row * p.ld_dkv, p.dkv_norm, rope, lane, [&](int c, const float2 x) { la_store2(dst + c, x); });
        __threadfence();
    }
    if (tid < LF_HEADS) {
        ml[tid] = -INFINITY;
        ml[LF_HEADS + tid] = 0.f;
    }
    for (int i = tid; i < LF_HEADS * po_ld; i += LA_THREADS) po[i] = 0.f;
    const float scale2 = p.scale * 1.4426950408889634f;
    for (int k0 = run.t0; k0 < run.t1; k0 += TK) {
        const int n = min(TK, run.t1 - k0);
        __syncthreads();
        run.load(kv, k0, TK, -1);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
        const int blocks = (n + 31) >> 5;
        for (int job = warp; job < nh * blocks; job += LA_WARPS) {
            const int h = job / blocks, k = (job - h * blocks) * 32 + lane;
            if (k < n) {
                float d = 0.f;
                for (int c = 0; c < W; c += 4) {
                    const float4 x = *reinterpret_cast<const float4*>(kv + (size_t)k * ws + c), q = *reinterpret_cast<const float4*>(qs + h * ws + c);
                    d += x.x * q.x + x.y * q.y + x.z * q.z + x.w * q.w;
                }
                sc[h * TK + k] = d * scale2;
            }
        }
        __syncthreads();
        for (int h = warp; h < nh; h += LA_WARPS) {
            float top = -INFINITY, sum = 0.f;
            for (int k = lane; k < n; k += 32) top = fmaxf(top, sc[h * TK + k]);
            const float m_old = ml[h], m_new = fmaxf(m_old, warp_max(top));
            for (int k = lane; k < n; k += 32) {
                const float e = exp2f(sc[h * TK + k] - m_new);
                sc[h * TK + k] = e;
                sum += e;
            }
            sum = warp_sum(sum);
            if (lane == 0) {
                const float al = exp2f(m_old - m_new);
                ml[h] = m_new;
                ml[LF_HEADS + h] = ml[LF_HEADS + h] * al + sum;
                ml[2 * LF_HEADS + h] = al;
            }
        }
        __syncthreads();
        for (int i = tid; i < nh * (s.kp >> 2); i += LA_THREADS) {  // (a thread's own sums: the same in every tile)
            const int h = i / (s.kp >> 2), c = (i - h * (s.kp >> 2)) * 4;
            float4* out = reinterpret_cast<float4*>(po + h * po_ld + c);
            const float al = ml[2 * LF_HEADS + h];
            float4 o = make_float4(out->x * al, out->y * al, out->z * al, out->w * al);
            for (int k = 0; k < n; ++k) {
                const float w = sc[h * TK + k];
                const float4 v = *reinterpret_cast<const float4*>(kv + (size_t)k * ws + c);
                o.x += w * v.x;
                o.y += w * v.y;
                o.z += w * v.z;
                o.w += w * v.w;
            }
            *out = o;
        }
    }
    la_merge<float>(p, po, po_ld, ml, LF_HEADS, h0, nh, run.row, rank, ns);
}

static size_t la_bytes(const LatentShape& s, int f32, int tile) {
    const size_t W = latent_row(s);
    if (f32) return sizeof(float) * (LF_HEADS * (W + 4) + tile * (W + 4) + LF_HEADS * tile + LF_HEADS * (s.kp + 4) + 3 * LF_HEADS);
    size_t kv = 2 * (size_t)tile * (W + 8) * 2;
    const size_t sums = (size_t)LA_HEADS * (s.kp + 4) * sizeof(float);
    if (kv < sums) return 0;
    return LA_HEADS * (W + 8) * 2 + kv + LA_HEADS * (size_t)(tile + 8) * 2 + 2 * LA_HEADS * (size_t)(tile + 4) * sizeof(float) + 3 * LA_HEADS * sizeof(float);
}
static int la_tile(const LatentShape& s, int f32) {
    for (int tile = 64; tile >= (f32 ? 8 : 16); tile >>= 1) {
        const size_t n = la_bytes(s, f32, tile);
        if (n && n <= LA_SMEM_MAX) return tile;
    }
    return 0;
}
bool latent_attn_supported(const LatentShape& s, int f32) {
    return s.heads > 0 && s.kp > 0 && s.rp >= 0 && s.kp % 16 == 0 && s.rp % 16 == 0 && (f32 || s.kp <= 1024) && la_tile(s, f32) > 0;
}

typedef void (*LatentKernel)(LatentArgs);
static LatentKernel la_kernel(const LatentShape& s, int f32) {
    if (f32) return latent_attn_f32_kernel;
    return s.kp <= 256 ? latent_attn_mma_kernel<1> : s.kp <= 512 ? latent_attn_mma_kernel<2> : latent_attn_mma_kernel<4>;
}

// Sets the kernels up; whether the device places clusters of sixteen of this one.
static int la_configure(LatentKernel kernel, size_t smem, bool* sixteen) {
    static PerDevice<bool> once;
    if (!once.here()) {
        for (LatentKernel k : {(LatentKernel)latent_attn_f32_kernel, (LatentKernel)latent_attn_mma_kernel<1>, (LatentKernel)latent_attn_mma_kernel<2>,
                               (LatentKernel)latent_attn_mma_kernel<4>}) {
            RB_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LA_SMEM_MAX));
            RB_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
        }
        once.here() = true;
    }
    struct Known {
        LatentKernel kernel;
        size_t smem;
        bool sixteen;
    };
    static PerDevice<Known> last;
    Known& known = last.here();
    if (known.kernel != kernel || known.smem != smem) {
        cudaLaunchConfig_t cfg = {};
        cfg.gridDim = dim3(LA_MAX_SPLITS);
        cfg.blockDim = dim3(LA_THREADS);
        cfg.dynamicSmemBytes = smem;
        cudaLaunchAttribute attr[1];
        attr[0].id = cudaLaunchAttributeClusterDimension;
        attr[0].val.clusterDim.x = LA_MAX_SPLITS;
        attr[0].val.clusterDim.y = 1;
        attr[0].val.clusterDim.z = 1;
        cfg.attrs = attr;
        cfg.numAttrs = 1;
        int clusters = 0;
        const bool ok = cudaOccupancyMaxActiveClusters(&clusters, kernel, &cfg) == cudaSuccess && clusters > 0;
        cudaGetLastError();
        known = {kernel, smem, ok};
    }
    *sixteen = known.sixteen;
    return ROTOR_B200_OK;
}

int launch_latent_attn(const LatentAttn& p, int rows, cudaStream_t st) {
    RB_REQUIRE(p.q_abs && p.cache.rows && p.cache.past_len && p.cache.rope && p.out && rows > 0 && p.cache.seq > 0);
    RB_REQUIRE(!p.dkv || (p.dkv_norm && p.cache.seq == 1));
    if (!latent_attn_supported(p.s, p.f32)) return ROTOR_B200_ERR_SHAPE;
    const int per = p.f32 ? LF_HEADS : LA_HEADS, head_tiles = (p.s.heads + per - 1) / per;
    const int reach = p.window > 0 && p.window < p.cache.max_seq ? p.window : p.cache.max_seq;
    LatentArgs a = {};
    a.p = p;
    a.tile = la_tile(p.s, p.f32);
    const size_t smem = la_bytes(p.s, p.f32, a.tile);
    const LatentKernel kernel = la_kernel(p.s, p.f32);
    bool sixteen;
    const int rc = la_configure(kernel, smem, &sixteen);
    if (rc) return rc;
    for (int r0 = 0; r0 < rows; r0 += 65535) {  // (the grid's z limit)
        const int n = rows - r0 < 65535 ? rows - r0 : 65535;
        const long long ctas = (long long)n * head_tiles;
        int splits = 1;
        while (splits < 8 && ctas * splits * 2 <= 148 && reach >= 32 * splits) splits *= 2;
        if (splits == 8 && sixteen && ctas <= 4 && reach >= 512) splits = 16;  // (a cluster of sixteen fills most of a GPC)
        a.row0 = r0;
        const int e = launch_chained(kernel, dim3(splits, head_tiles, n), dim3(LA_THREADS), smem, st, splits, a);
        if (e) return e;
    }
    return ROTOR_B200_OK;
}

}  // namespace rb

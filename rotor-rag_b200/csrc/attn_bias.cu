// Softmax attention with a distance bias and a chunk mask, one query position at a time:
//   score(i, j) = (q_i . k_j) scale - slope_h (i - j),   j <= i, with chunks of C j / C == i / C, with a window of
// N i - j < N, and a sink per head in the softmax's denominator.
// Used by generation steps (one token per sequence; the new key and value are normalised and appended
// here), by short portions, by float32 runs, and by head sizes the tensor-core kernel does not take.
//
// Grid (splits, KV heads x head blocks, rows); the splits of a row form a thread-block cluster.  A CTA
// takes an equal run of the row's visible keys for the query heads of one group, walks it in tiles
// staged by cp.async (the first tile is requested before the programmatic-launch wait: it holds only
// rows that earlier steps appended), keeps a running maximum and sum per head, and the cluster merges
// its partial outputs through distributed shared memory.
#include "decoder.cuh"

namespace rb {

constexpr int BA_THREADS = 256, BA_WARPS = BA_THREADS / 32;
constexpr int BA_MAX_SPLITS = 8;
constexpr int BA_MAX_PAIRS = 16;            // output column pairs per thread
constexpr size_t BA_SMEM_MAX = 200 * 1024;

struct BiasRowsArgs {
    BiasAttn p;
    int row0;                           // first row of this launch
    int tile, head_block, head_blocks;  // keys per staged tile; query heads per CTA; CTAs per group
};

__device__ __forceinline__ uint32_t ba_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ float ba_ld_cluster(const float* local, unsigned rank) {
    uint32_t a;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(ba_smem(local)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(a) : "memory");
    return v;
}
template <typename T>
__device__ __forceinline__ void ba_load8(const T* p, float (&f)[8]);
template <>
__device__ __forceinline__ void ba_load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&f)[8]) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const float4 a = bf16x4_to_float4(make_uint2(u.x, u.y)), b = bf16x4_to_float4(make_uint2(u.z, u.w));
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
template <>
__device__ __forceinline__ void ba_load8<float>(const float* p, float (&f)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ float2 ba_load2(const __nv_bfloat16* p) {
    const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
    return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
}
__device__ __forceinline__ float2 ba_load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ void ba_store(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void ba_store(float* p, float v) { *p = v; }
__device__ __forceinline__ float ba_round(float v, const __nv_bfloat16*) { return round_bf16(v); }
__device__ __forceinline__ float ba_round(float v, const float*) { return v; }

// Merges the cluster's runs, every CTA a share of the outputs.  po: this CTA's un-normalised output
// [heads][stride], ml: maxima [heads][1], sums at ml + HB.  All threads of the CTA call.
template <typename T>
__device__ __forceinline__ void ba_merge(const BiasAttn& p, const float* po, int stride, const float* ml, int HB, int nh, int head0,
                                         int row, int rank, int ns, int tid, int nthr, const T*) {
    if (ns > 1)
        asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
    else
        __syncthreads();
    const int vdim = p.s.vdim;
    T* out = static_cast<T*>(p.out) + (size_t)row * p.ld_out;
    const int total = nh * vdim;
    for (int idx = rank * nthr + tid; idx < total; idx += ns * nthr) {
        const int h = idx / vdim, c = idx - h * vdim;
        const float sink = p.sinks ? __ldg(p.sinks + head0 + h) * 1.4426950408889634f : -INFINITY;
        float o, l, M = sink;
        if (ns == 1) {
            o = po[h * stride + c];
            l = ml[HB + h];
            if (p.sinks) {
                M = fmaxf(M, ml[h]);
                const float e = exp2f(ml[h] - M);
                o *= e;
                l *= e;
            }
        } else {
            float m[BA_MAX_SPLITS], w[BA_MAX_SPLITS], v[BA_MAX_SPLITS];
#pragma unroll
            for (int k = 0; k < BA_MAX_SPLITS; ++k) {  // (all remote reads in flight together)
                m[k] = k < ns ? ba_ld_cluster(ml + h, k) : -INFINITY;
                w[k] = k < ns ? ba_ld_cluster(ml + HB + h, k) : 0.f;
                v[k] = k < ns ? ba_ld_cluster(po + h * stride + c, k) : 0.f;
            }
#pragma unroll
            for (int k = 0; k < BA_MAX_SPLITS; ++k) M = fmaxf(M, m[k]);
            o = 0.f;
            l = 0.f;
#pragma unroll
            for (int k = 0; k < BA_MAX_SPLITS; ++k) {
                const float e = exp2f(m[k] - M);
                l += e * w[k];
                o += e * v[k];
            }
        }
        if (p.sinks) l += exp2f(sink - M);
        ba_store(out + (size_t)(head0 + h) * vdim + c, o / l);
    }
    if (ns > 1)  // nobody leaves while its shared memory may still be read
        asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

template <typename T, int NI>
__global__ void __launch_bounds__(BA_THREADS) bias_attn_rows_kernel(const __grid_constant__ BiasRowsArgs a) {
    const BiasAttn& p = a.p;
    const HeadShape& s = p.s;
    extern __shared__ __align__(16) unsigned char ba_raw[];
    constexpr int PAD = 16 / (int)sizeof(T);
    const int R = s.heads / s.kv_heads, HB = a.head_block, TK = a.tile;
    const int ks = s.kd + PAD, vs = s.vd + PAD;  // staged row strides: 128-bit column reads without bank conflicts
    float* qs = reinterpret_cast<float*>(ba_raw);           // [HB][kd]
    float* ps = qs + HB * s.kd;                             // [HB][TK]
    float* ml = ps + HB * TK;                               // m [HB], l [HB], alpha [HB]
    float* po = ml + ((3 * HB + 3) & ~3);                   // [HB][vd] this CTA's partial output
    T* kn = reinterpret_cast<T*>(po + HB * s.vd);           // [kd], [vd]: the appended key and value
    T* vn = kn + s.kd;
    T* Ks = vn + s.vd;                                      // [2][TK][ks]
    T* Vs = Ks + 2 * TK * ks;                               // [2][TK][vs]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int ns = (int)gridDim.x, rank = (int)blockIdx.x;
    const int hk = (int)blockIdx.y / a.head_blocks, h0 = ((int)blockIdx.y - hk * a.head_blocks) * HB;
    const int nh = min(HB, R - h0);                         // query heads of this CTA: hk R + h0 ..
    const int row = a.row0 + (int)blockIdx.z, b = row / p.cache.seq;
    const int pos = min(cached_len(p.cache.past_len, b, p.cache.max_seq) + (row - b * p.cache.seq), p.cache.max_seq - 1);
    const int lo = first_visible(pos, p.chunk, p.window);
    const int per = (pos + 1 - lo + ns - 1) / ns;
    const int t0 = lo + rank * per, t1 = min(t0 + per, pos + 1);
    const size_t head_row = ((size_t)b * s.kv_heads + hk) * p.cache.max_seq;
    T* kc = static_cast<T*>(p.cache.k) + head_row * s.kd;
    T* vc = static_cast<T*>(p.cache.v) + head_row * s.vd;
    const int kch = s.kd / (16 / (int)sizeof(T)), vch = s.vd / (16 / (int)sizeof(T));  // 16-byte pieces per row

    auto load_tile = [&](int k0, int buf) {
        const int n = min(TK, t1 - k0);
        for (int i = tid; i < n * (kch + vch); i += BA_THREADS) {
            const int j = i / (kch + vch), c = i - j * (kch + vch);
            if (p.append && k0 + j == pos) continue;
            const bool isv = c >= kch;
            const void* src = isv ? (const void*)(vc + (size_t)(k0 + j) * s.vd + (c - kch) * PAD) : (const void*)(kc + (size_t)(k0 + j) * s.kd + c * PAD);
            const uint32_t dst = isv ? ba_smem(Vs + (size_t)(buf * TK + j) * vs + (c - kch) * PAD) : ba_smem(Ks + (size_t)(buf * TK + j) * ks + c * PAD);
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (t0 < t1) load_tile(t0, 0);
    pdl_wait();
    pdl_trigger();

    // ---- queries (normalised), the new key and value
    const float* raw = p.qkv + (size_t)row * p.ld_qkv;
    auto inv_rms = [&](const float* v) {
        if (!s.unit) return 1.f;
        float ss = 0.f;
        for (int c = lane; c < s.dim; c += 32) {
            const float x = __ldcg(v + c);
            ss += x * x;
        }
        return 1.0f / sqrtf(warp_sum(ss) / (float)s.dim + s.eps);
    };
    for (int h = warp; h < nh; h += BA_WARPS) {
        const float* v = raw + (size_t)(hk * R + h0 + h) * s.dim;
        const float inv = inv_rms(v);
        for (int c = lane; c < s.kd; c += 32) qs[h * s.kd + c] = c < s.dim ? ba_round(__ldcg(v + c) * inv, kc) : 0.f;
    }
    const bool owner = p.append && t0 <= pos && pos < t1;  // (the last key of the run)
    if (owner && warp == BA_WARPS - 1) {
        const float* v = raw + (size_t)(s.heads + hk) * s.dim;
        const float inv = inv_rms(v);
        for (int c = lane; c < s.kd; c += 32) {
            const float x = c < s.dim ? __ldcg(v + c) * inv : 0.f;
            ba_store(kn + c, x);
            if (h0 == 0) ba_store(kc + (size_t)pos * s.kd + c, x);
        }
    } else if (owner && warp == BA_WARPS - 2) {
        const float* v = raw + (size_t)(s.heads + s.kv_heads) * s.dim + (size_t)hk * s.vdim;
        for (int c = lane; c < s.vd; c += 32) {
            const float x = c < s.vdim ? __ldcg(v + c) : 0.f;
            ba_store(vn + c, x);
            if (h0 == 0) ba_store(vc + (size_t)pos * s.vd + c, x);
        }
    }
    for (int h = tid; h < HB; h += BA_THREADS) {
        ml[h] = -INFINITY;
        ml[HB + h] = 0.f;
    }

    float2 acc[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) acc[i] = make_float2(0.f, 0.f);
    const int vp = s.vd >> 1, items = nh * vp;
    const float scale2 = p.scale * 1.4426950408889634f;
    for (int k0 = t0, it = 0; k0 < t1; k0 += TK, ++it) {
        const int buf = it & 1, n = min(TK, t1 - k0);
        if (k0 + TK < t1) {
            __syncthreads();  // the other buffer's readers are done
            load_tile(k0 + TK, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        if (owner && k0 + n == pos + 1) {  // the new row's place in its tile (the lanes that made it copy it)
            if (warp == BA_WARPS - 1)
                for (int c = lane; c < s.kd; c += 32) Ks[(size_t)(buf * TK + n - 1) * ks + c] = kn[c];
            else if (warp == BA_WARPS - 2)
                for (int c = lane; c < s.vd; c += 32) Vs[(size_t)(buf * TK + n - 1) * vs + c] = vn[c];
        }
        __syncthreads();
        const int blocks = (n + 31) >> 5;
        for (int job = warp; job < nh * blocks; job += BA_WARPS) {
            const int h = job / blocks, key = (job - h * blocks) * 32 + lane;
            float sc = -INFINITY;
            if (key < n) {
                const T* kr = Ks + (size_t)(buf * TK + key) * ks;
                const float* q = qs + h * s.kd;
                float d = 0.f;
                for (int c = 0; c < s.kd; c += 8) {
                    float f[8];
                    ba_load8<T>(kr + c, f);
                    const float4 qa = *reinterpret_cast<const float4*>(q + c), qb = *reinterpret_cast<const float4*>(q + c + 4);
                    d += f[0] * qa.x;
                    d += f[1] * qa.y;
                    d += f[2] * qa.z;
                    d += f[3] * qa.w;
                    d += f[4] * qb.x;
                    d += f[5] * qb.y;
                    d += f[6] * qb.z;
                    d += f[7] * qb.w;
                }
                const float slope = p.slopes ? __ldg(p.slopes + hk * R + h0 + h) : 0.f;
                sc = d * scale2 - slope * 1.4426950408889634f * (float)(pos - (k0 + key));
            }
            ps[h * TK + key] = sc;
        }
        __syncthreads();
        for (int h = warp; h < nh; h += BA_WARPS) {
            float tm = -INFINITY;
            for (int key = lane; key < n; key += 32) tm = fmaxf(tm, ps[h * TK + key]);
            const float m_old = ml[h], m_new = fmaxf(m_old, warp_max(tm));  // finite: every key of the run is visible
            float sum = 0.f;
            for (int key = lane; key < n; key += 32) {
                const float e = exp2f(ps[h * TK + key] - m_new);
                ps[h * TK + key] = e;
                sum += e;
            }
            sum = warp_sum(sum);
            if (lane == 0) {
                const float al = exp2f(m_old - m_new);
                ml[h] = m_new;
                ml[HB + h] = ml[HB + h] * al + sum;
                ml[2 * HB + h] = al;
            }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int idx = tid + i * BA_THREADS;
            if (idx < items) {
                const int h = idx / vp, c = (idx - h * vp) * 2;
                const float al = ml[2 * HB + h];
                float2 o = make_float2(acc[i].x * al, acc[i].y * al);
                const T* vr = Vs + (size_t)(buf * TK) * vs + c;
                const float* pr = ps + h * TK;
                int k = 0;
                for (; k + 4 <= n; k += 4) {
                    const float4 w = *reinterpret_cast<const float4*>(pr + k);
                    const float2 v0 = ba_load2(vr + (size_t)k * vs), v1 = ba_load2(vr + (size_t)(k + 1) * vs),
                                 v2 = ba_load2(vr + (size_t)(k + 2) * vs), v3 = ba_load2(vr + (size_t)(k + 3) * vs);
                    o.x += w.x * v0.x;
                    o.y += w.x * v0.y;
                    o.x += w.y * v1.x;
                    o.y += w.y * v1.y;
                    o.x += w.z * v2.x;
                    o.y += w.z * v2.y;
                    o.x += w.w * v3.x;
                    o.y += w.w * v3.y;
                }
                for (; k < n; ++k) {
                    const float2 v = ba_load2(vr + (size_t)k * vs);
                    o.x += pr[k] * v.x;
                    o.y += pr[k] * v.y;
                }
                acc[i] = o;
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int idx = tid + i * BA_THREADS;
        if (idx < items) {
            const int h = idx / vp, c = (idx - h * vp) * 2;
            *reinterpret_cast<float2*>(po + h * s.vd + c) = acc[i];
        }
    }
    ba_merge(p, po, s.vd, ml, HB, nh, hk * R + h0, row, rank, ns, tid, BA_THREADS, (const T*)nullptr);
}

// The same for head sizes up to 128 (64): a warp takes a strip of keys for all H query heads of its CTA
// and needs no shared memory until the end.  W lanes hold four columns each of a key and of the queries
// (W = 16: the two halves of the warp take alternate keys); keys come eight per half at a time, straight
// into registers, a batch ahead of the arithmetic.  The 8 H partial dot products are summed across the W
// lanes by a halving exchange (each step trades half of the values with the partner lane, so that every
// lane ends with its own scores instead of all of them), the softmax runs on those, and the weights are
// handed out again by shuffles.  Strips are folded in shared memory, CTAs of a cluster as above.
constexpr int BS_U = 8;  // keys per half and batch

__device__ __forceinline__ float4 bs_widen(const uint2 u, const __nv_bfloat16*) { return bf16x4_to_float4(u); }
__device__ __forceinline__ float4 bs_widen(const float4 v, const float*) { return v; }
__device__ __forceinline__ uint2 bs_narrow(const float4 v, const __nv_bfloat16*) { return float4_to_bf16x4(v); }
__device__ __forceinline__ float4 bs_narrow(const float4 v, const float*) { return v; }
template <typename T> struct BsVec;
template <> struct BsVec<__nv_bfloat16> { typedef uint2 type; };
template <> struct BsVec<float> { typedef float4 type; };

template <typename T, int W, int H, int NW>
__global__ void __launch_bounds__(32 * NW, sizeof(T) == 2 ? 16 / NW : 1) bias_attn_strips_kernel(const __grid_constant__ BiasRowsArgs a) {
    const BiasAttn& p = a.p;
    const HeadShape& s = p.s;
    constexpr int C = 4 * W, N = BS_U * H, VPL = N >= W ? N / W : 1, DUP = N >= W ? 1 : W / N, HALVES = 32 / W;
    typedef typename BsVec<T>::type Vec;
    __shared__ __align__(16) float part[NW][H][C];
    __shared__ float wml[2][NW][H], ml[2 * H];
    const int R = s.heads / s.kv_heads;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l = lane & (W - 1), half = lane / W, base = half * W;
    const int ns = (int)gridDim.x, rank = (int)blockIdx.x;
    const int hk = (int)blockIdx.y / a.head_blocks, h0 = ((int)blockIdx.y - hk * a.head_blocks) * H;
    const int nh = min(H, R - h0);
    const int row = a.row0 + (int)blockIdx.z, b = row / p.cache.seq;
    const int pos = min(cached_len(p.cache.past_len, b, p.cache.max_seq) + (row - b * p.cache.seq), p.cache.max_seq - 1);
    const int lo = first_visible(pos, p.chunk, p.window);
    const int cached = pos + (p.append ? 0 : 1) - lo;  // keys read from the cache
    // the very last warp takes the new key, the others share the cached ones
    const int strips = ns * NW - (p.append ? 1 : 0), per = (cached + strips - 1) / strips;
    const int a0 = lo + (rank * NW + warp) * per, a1 = min(a0 + per, lo + cached);  // (empty for the last warp)
    const size_t head_row = ((size_t)b * s.kv_heads + hk) * p.cache.max_seq;
    T* kc = static_cast<T*>(p.cache.k) + head_row * s.kd;
    T* vc = static_cast<T*>(p.cache.v) + head_row * s.vd;
    const bool kon = 4 * l < s.kd, von = 4 * l < s.vd;

    Vec kv[BS_U], vv[BS_U];
    auto fetch_k = [&](int j0) {
#pragma unroll
        for (int u = 0; u < BS_U; ++u) {
            const int j = j0 + u * HALVES + half;
            kv[u] = Vec{};
            if (j < a1 && kon) kv[u] = *reinterpret_cast<const Vec*>(kc + (size_t)j * s.kd + 4 * l);
        }
    };
    auto fetch_v = [&](int j0) {
#pragma unroll
        for (int u = 0; u < BS_U; ++u) {
            const int j = j0 + u * HALVES + half;
            vv[u] = Vec{};
            if (j < a1 && von) vv[u] = *reinterpret_cast<const Vec*>(vc + (size_t)j * s.vd + 4 * l);
        }
    };
    fetch_k(a0);
    fetch_v(a0);
    pdl_wait();
    pdl_trigger();

    // ---- this lane's four columns of every query, divided by the row's root mean square
    const float* raw = p.qkv + (size_t)row * p.ld_qkv;
    const bool vec = ((s.dim | s.vdim | p.ld_qkv) & 3) == 0;
    auto load_raw = [&](const float* v, int len) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (vec) {  // rows start on 16 bytes
            if (4 * l < len) x = __ldcg(reinterpret_cast<const float4*>(v + 4 * l));
            return x;
        }
        if (4 * l < len) x.x = __ldcg(v + 4 * l);
        if (4 * l + 1 < len) x.y = __ldcg(v + 4 * l + 1);
        if (4 * l + 2 < len) x.z = __ldcg(v + 4 * l + 2);
        if (4 * l + 3 < len) x.w = __ldcg(v + 4 * l + 3);
        return x;
    };
    auto finish = [&](float4 x, bool norm) {
        float inv = 1.f;
        if (norm) {
            float ss = x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
#pragma unroll
            for (int m = W / 2; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
            inv = 1.0f / sqrtf(ss / (float)s.dim + s.eps);
        }
        return make_float4(ba_round(x.x * inv, kc), ba_round(x.y * inv, kc), ba_round(x.z * inv, kc), ba_round(x.w * inv, kc));
    };
    float4 q[H];
#pragma unroll
    for (int h = 0; h < H; ++h) q[h] = h < nh ? load_raw(raw + (size_t)(hk * R + h0 + h) * s.dim, s.dim) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int h = 0; h < H; ++h) q[h] = finish(q[h], s.unit);

    const float scale2 = p.scale * 1.4426950408889634f;
    const int my_h = (VPL * l / DUP) >> 3;               // the head of this lane's scores
    const float slope2 = p.slopes && my_h < nh ? __ldg(p.slopes + hk * R + h0 + my_h) * 1.4426950408889634f : 0.f;
    float m_run = -INFINITY, l_run = 0.f;                // of head my_h; l_run over this lane's own scores
    float4 o[H];
#pragma unroll
    for (int h = 0; h < H; ++h) o[h] = make_float4(0.f, 0.f, 0.f, 0.f);

    // scores of a batch (sc: partial dot products, index h * 8 + u) -> weights; then O += weights V
    auto batch = [&](float (&sc)[N], int j0, int end) {
#pragma unroll
        for (int m = W / 2, cnt = N; m > 0; m >>= 1) {
            if (cnt > 1) {
                cnt >>= 1;
#pragma unroll
                for (int i = 0; i < N / 2; ++i)
                    if (i < cnt) {
                        const bool up = lane & m;
                        const float send = up ? sc[i] : sc[i + cnt], keep = up ? sc[i + cnt] : sc[i];
                        sc[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
                    }
            } else {
                sc[0] += __shfl_xor_sync(0xffffffffu, sc[0], m);
            }
        }
        float top = -INFINITY;
#pragma unroll
        for (int i = 0; i < VPL; ++i) {
            const int u = (VPL * l / DUP + i) & 7, j = j0 + u * HALVES + half;
            sc[i] = j < end ? sc[i] * scale2 - slope2 * (float)(pos - j) : -INFINITY;
            top = fmaxf(top, sc[i]);
        }
#pragma unroll
        for (int m = W / H / 2; m > 0; m >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, m));
        if (HALVES == 2) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 16));
        const float m_new = fmaxf(m_run, top), alpha = exp2f(m_run - m_new);  // (finite: a batch has a key)
        m_run = m_new;
        l_run *= alpha;
#pragma unroll
        for (int i = 0; i < VPL; ++i) {
            sc[i] = exp2f(sc[i] - m_new);
            l_run += sc[i];
        }
#pragma unroll
        for (int h = 0; h < H; ++h) {
            const float al = __shfl_sync(0xffffffffu, alpha, base + h * (W / H));
            o[h] = make_float4(o[h].x * al, o[h].y * al, o[h].z * al, o[h].w * al);
        }
#pragma unroll
        for (int u = 0; u < BS_U; ++u) {
            const float4 v = bs_widen(vv[u], kc);
#pragma unroll
            for (int h = 0; h < H; ++h) {
                const int idx = h * 8 + u;
                const float w = __shfl_sync(0xffffffffu, sc[VPL > 1 ? idx % VPL : 0], base + (VPL > 1 ? idx / VPL : idx * DUP));
                o[h].x += w * v.x;
                o[h].y += w * v.y;
                o[h].z += w * v.z;
                o[h].w += w * v.w;
            }
        }
    };
    for (int j0 = a0; j0 < a1; j0 += BS_U * HALVES) {
        float sc[N];
#pragma unroll
        for (int u = 0; u < BS_U; ++u) {
            const float4 k = bs_widen(kv[u], kc);
#pragma unroll
            for (int h = 0; h < H; ++h) sc[h * 8 + u] = k.x * q[h].x + k.y * q[h].y + k.z * q[h].z + k.w * q[h].w;
        }
        fetch_k(j0 + BS_U * HALVES);
        batch(sc, j0, a1);
        fetch_v(j0 + BS_U * HALVES);
    }
    if (p.append && rank == ns - 1 && warp == NW - 1) {  // the new key and value
        const float4 k = finish(load_raw(raw + (size_t)(s.heads + hk) * s.dim, s.dim), s.unit);
        const float4 v = finish(load_raw(raw + (size_t)(s.heads + s.kv_heads) * s.dim + (size_t)hk * s.vdim, s.vdim), false);
        if (h0 == 0 && half == 0) {
            const float kf[4] = {k.x, k.y, k.z, k.w}, vf[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                if (kon) ba_store(kc + (size_t)pos * s.kd + 4 * l + e, kf[e]);
                if (von) ba_store(vc + (size_t)pos * s.vd + 4 * l + e, vf[e]);
            }
        }
        float sc[N];
#pragma unroll
        for (int u = 0; u < BS_U; ++u) vv[u] = u == 0 && half == 0 ? bs_narrow(v, kc) : Vec{};
#pragma unroll
        for (int h = 0; h < H; ++h)
#pragma unroll
            for (int u = 0; u < BS_U; ++u)
                sc[h * 8 + u] = u == 0 ? k.x * q[h].x + k.y * q[h].y + k.z * q[h].z + k.w * q[h].w : 0.f;
        batch(sc, pos, pos + 1);
    }

    // ---- fold the strips
#pragma unroll
    for (int m = W / H / 2; m > 0; m >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, m);
    l_run *= 1.0f / DUP;
    if (HALVES == 2) l_run += __shfl_xor_sync(0xffffffffu, l_run, 16);
#pragma unroll
    for (int h = 0; h < H; ++h) {
        if (HALVES == 2) {
            o[h].x += __shfl_xor_sync(0xffffffffu, o[h].x, 16);
            o[h].y += __shfl_xor_sync(0xffffffffu, o[h].y, 16);
            o[h].z += __shfl_xor_sync(0xffffffffu, o[h].z, 16);
            o[h].w += __shfl_xor_sync(0xffffffffu, o[h].w, 16);
        }
        if (half == 0) *reinterpret_cast<float4*>(&part[warp][h][4 * l]) = o[h];
    }
    if (half == 0 && l % (W / H) == 0) {
        wml[0][warp][my_h] = m_run;
        wml[1][warp][my_h] = l_run;
    }
    __syncthreads();
    for (int i = tid; i < H * C; i += 32 * NW) {
        const int h = i / C, c = i - h * C;
        float M = -INFINITY, t = 0.f, sum = 0.f;
#pragma unroll
        for (int w = 0; w < NW; ++w) M = fmaxf(M, wml[0][w][h]);
        if (M > -INFINITY) {
#pragma unroll
            for (int w = 0; w < NW; ++w) {
                const float e = exp2f(wml[0][w][h] - M);
                t += e * part[w][h][c];
                sum += e * wml[1][w][h];
            }
        }
        part[0][h][c] = t;  // (element read by this thread alone)
        if (c == 0) {
            ml[h] = M;
            ml[H + h] = sum;
        }
    }
    ba_merge(p, &part[0][0][0], C, ml, H, nh, hk * R + h0, row, rank, ns, tid, 32 * NW, (const T*)nullptr);
}

int bias_attn_reach(const BiasAttn& p) {
    int reach = p.cache.max_seq;
    if (p.chunk > 0 && p.chunk < reach) reach = p.chunk;
    if (p.window > 0 && p.window < reach) reach = p.window;
    return reach;
}

template <typename T>
static size_t ba_smem_bytes(const HeadShape& s, int hb, int tile) {
    const size_t pad = 16 / sizeof(T);
    return sizeof(float) * ((size_t)hb * s.kd + (size_t)hb * tile + ((3 * hb + 3) & ~3) + (size_t)hb * s.vd) +
           sizeof(T) * (2 * (size_t)tile * (s.kd + pad + s.vd + pad) + s.kd + s.vd);
}

template <typename K>
static int ba_go(K kernel, const BiasRowsArgs& a, int rows, int splits, size_t smem, cudaStream_t st, int threads = BA_THREADS) {
    const dim3 grid(splits, a.p.s.kv_heads * a.head_blocks, rows);
    if (a.p.append) return launch_chained(kernel, grid, dim3(threads), smem, st, splits, a);
    // (rows appended by the kernel just before: no early start)
    const int pdl = g_use_pdl;
    g_use_pdl = 0;
    const int rc = launch_chained(kernel, grid, dim3(threads), smem, st, splits, a);
    g_use_pdl = pdl;
    return rc;
}

template <typename T, int NI>
static int ba_launch(const BiasRowsArgs& a, int rows, int splits, size_t smem, cudaStream_t st) {
    static PerDevice<bool> once;
    if (!once.here()) {
        RB_CUDA(cudaFuncSetAttribute(bias_attn_rows_kernel<T, NI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)BA_SMEM_MAX));
        once.here() = true;
    }
    return ba_go(bias_attn_rows_kernel<T, NI>, a, rows, splits, smem, st);
}

template <typename T, int W, int NW>
static int bs_launch(const BiasRowsArgs& a, int h, int rows, int splits, cudaStream_t st) {
    switch (h) {
        case 1: return ba_go(bias_attn_strips_kernel<T, W, 1, NW>, a, rows, splits, 0, st, 32 * NW);
        case 2: return ba_go(bias_attn_strips_kernel<T, W, 2, NW>, a, rows, splits, 0, st, 32 * NW);
        default: return ba_go(bias_attn_strips_kernel<T, W, 4, NW>, a, rows, splits, 0, st, 32 * NW);
    }
}
template <typename T, int W>
static int bs_pick(const BiasRowsArgs& a, int h, int rows, int splits, int reach, cudaStream_t st) {
    // few CTAs and long runs: twice the warps per CTA
    if constexpr (sizeof(T) == 2)
        if ((long long)rows * a.p.s.kv_heads * a.head_blocks * splits <= 148 && reach >= 128 * splits)
            return bs_launch<T, W, 16>(a, h, rows, splits, st);
    return bs_launch<T, W, 8>(a, h, rows, splits, st);
}

static int ba_splits(long long ctas, int reach) {
    // (clusters of eight do not fill every GPC: beyond about a hundred CTAs some would wait for a second round)
    int splits = 1;
    while (splits < BA_MAX_SPLITS && ctas * splits * 2 <= (splits == 4 ? 96 : 148) && reach >= 64 * splits) splits *= 2;
    return splits;
}

template <typename T>
static int ba_pick(const BiasAttn& p, int row0, int rows, cudaStream_t st) {
    const HeadShape& s = p.s;
    BiasRowsArgs a = {};
    a.p = p;
    a.row0 = row0;
    const int R = s.heads / s.kv_heads, vp = s.vd / 2, reach = bias_attn_reach(p);
    if (s.kd <= 128 && s.vd <= 128) {
        int h = 1;
        while (h < R && h < 4) h *= 2;
        a.head_block = h;
        a.head_blocks = (R + h - 1) / h;
        if (s.kv_heads * a.head_blocks > 65535) return ROTOR_B200_ERR_SHAPE;
        const int splits = ba_splits((long long)rows * s.kv_heads * a.head_blocks, reach);
        return s.kd <= 64 && s.vd <= 64 ? bs_pick<T, 16>(a, h, rows, splits, reach, st) : bs_pick<T, 32>(a, h, rows, splits, reach, st);
    }
    a.head_block = R;
    const int most = BA_MAX_PAIRS * BA_THREADS / vp;
    if (most < 1) return ROTOR_B200_ERR_SHAPE;
    if (a.head_block > most) a.head_block = most;
    a.tile = 128;
    for (;;) {
        while (a.tile > 32 && ba_smem_bytes<T>(s, a.head_block, a.tile) > BA_SMEM_MAX) a.tile >>= 1;
        if (ba_smem_bytes<T>(s, a.head_block, a.tile) <= BA_SMEM_MAX) break;
        if (a.head_block == 1) return ROTOR_B200_ERR_SHAPE;
        a.head_block = (a.head_block + 1) / 2;
    }
    a.head_blocks = (R + a.head_block - 1) / a.head_block;
    const long long ctas = (long long)rows * s.kv_heads * a.head_blocks;
    const int splits = ba_splits(ctas, reach);
    // a run shorter than the tile needs no larger tile
    const int run = (reach + splits - 1) / splits;
    while (a.tile > 32 && run <= a.tile / 2) a.tile >>= 1;
    const size_t smem = ba_smem_bytes<T>(s, a.head_block, a.tile);
    if (s.kv_heads * a.head_blocks > 65535) return ROTOR_B200_ERR_SHAPE;
    const int pairs = (a.head_block * vp + BA_THREADS - 1) / BA_THREADS;
    if (pairs <= 1) return ba_launch<T, 1>(a, rows, splits, smem, st);
    if (pairs <= 2) return ba_launch<T, 2>(a, rows, splits, smem, st);
    if (pairs <= 4) return ba_launch<T, 4>(a, rows, splits, smem, st);
    if (pairs <= 8) return ba_launch<T, 8>(a, rows, splits, smem, st);
    return ba_launch<T, BA_MAX_PAIRS>(a, rows, splits, smem, st);
}

int launch_bias_attn_rows(const BiasAttn& p, int rows, cudaStream_t st) {
    RB_REQUIRE(p.qkv && p.cache.k && p.cache.v && p.cache.past_len && p.out && rows > 0 && p.cache.seq > 0);
    RB_REQUIRE(!p.append || p.cache.seq == 1);
    RB_REQUIRE(p.s.heads % p.s.kv_heads == 0 && p.s.kd % 8 == 0 && p.s.vd % 8 == 0);
    for (int r0 = 0; r0 < rows; r0 += 65535) {  // (the grid's z limit)
        const int n = rows - r0 < 65535 ? rows - r0 : 65535;
        const int rc = p.f32 ? ba_pick<float>(p, r0, n, st) : ba_pick<__nv_bfloat16>(p, r0, n, st);
        if (rc) return rc;
    }
    return ROTOR_B200_OK;
}

}  // namespace rb

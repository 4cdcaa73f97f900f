// Softmax attention with a distance bias and a chunk mask, one query position at a time:
//   score(i, j) = (q_i . k_j) scale - slope_h (i - j),   j <= i and, with chunks of C, j / C == i / C.
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
    const int pos = min(p.cache.past_len[b] + (row - b * p.cache.seq), p.cache.max_seq - 1);
    const int lo = p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
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
    // ---- merge the cluster's runs: this CTA writes every ns-th output
    if (ns > 1)
        asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
    else
        __syncthreads();
    T* out = static_cast<T*>(p.out) + (size_t)row * p.ld_out;
    const int total = nh * s.vdim;
    for (int idx = rank * BA_THREADS + tid; idx < total; idx += ns * BA_THREADS) {
        const int h = idx / s.vdim, c = idx - h * s.vdim;
        float o, l;
        if (ns == 1) {
            o = po[h * s.vd + c];
            l = ml[HB + h];
        } else {
            float m[BA_MAX_SPLITS], M = -INFINITY;
            for (int k = 0; k < BA_MAX_SPLITS; ++k) {
                m[k] = k < ns ? ba_ld_cluster(ml + h, k) : -INFINITY;
                M = fmaxf(M, m[k]);
            }
            o = 0.f;
            l = 0.f;
            for (int k = 0; k < BA_MAX_SPLITS; ++k)
                if (k < ns) {
                    const float w = exp2f(m[k] - M);
                    l += w * ba_ld_cluster(ml + HB + h, k);
                    o += w * ba_ld_cluster(po + h * s.vd + c, k);
                }
        }
        ba_store(out + (size_t)(hk * R + h0 + h) * s.vdim + c, o / l);
    }
    if (ns > 1)  // nobody leaves while its shared memory may still be read
        asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

int bias_attn_reach(const BiasAttn& p) {
    return p.chunk > 0 && p.chunk < p.cache.max_seq ? p.chunk : p.cache.max_seq;
}

template <typename T>
static size_t ba_smem_bytes(const HeadShape& s, int hb, int tile) {
    const size_t pad = 16 / sizeof(T);
    return sizeof(float) * ((size_t)hb * s.kd + (size_t)hb * tile + ((3 * hb + 3) & ~3) + (size_t)hb * s.vd) +
           sizeof(T) * (2 * (size_t)tile * (s.kd + pad + s.vd + pad) + s.kd + s.vd);
}

template <typename T, int NI>
static int ba_launch(const BiasRowsArgs& a, int rows, int splits, size_t smem, cudaStream_t st) {
    static PerDevice<bool> once;
    if (!once.here()) {
        RB_CUDA(cudaFuncSetAttribute(bias_attn_rows_kernel<T, NI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)BA_SMEM_MAX));
        once.here() = true;
    }
    const dim3 grid(splits, a.p.s.kv_heads * a.head_blocks, rows);
    if (a.p.append) return launch_chained(bias_attn_rows_kernel<T, NI>, grid, dim3(BA_THREADS), smem, st, splits, a);
    // (rows appended by the kernel just before: no early start)
    const int pdl = g_use_pdl;
    g_use_pdl = 0;
    const int rc = launch_chained(bias_attn_rows_kernel<T, NI>, grid, dim3(BA_THREADS), smem, st, splits, a);
    g_use_pdl = pdl;
    return rc;
}

template <typename T>
static int ba_pick(const BiasAttn& p, int row0, int rows, cudaStream_t st) {
    const HeadShape& s = p.s;
    BiasRowsArgs a = {};
    a.p = p;
    a.row0 = row0;
    const int R = s.heads / s.kv_heads, vp = s.vd / 2;
    a.head_block = R;
    const int most = BA_MAX_PAIRS * BA_THREADS / vp;
    if (most < 1) return ROTOR_B200_ERR_SHAPE;
    if (a.head_block > most) a.head_block = most;
    const int reach = bias_attn_reach(p);
    a.tile = 128;
    for (;;) {
        while (a.tile > 32 && ba_smem_bytes<T>(s, a.head_block, a.tile) > BA_SMEM_MAX) a.tile >>= 1;
        if (ba_smem_bytes<T>(s, a.head_block, a.tile) <= BA_SMEM_MAX) break;
        if (a.head_block == 1) return ROTOR_B200_ERR_SHAPE;
        a.head_block = (a.head_block + 1) / 2;
    }
    a.head_blocks = (R + a.head_block - 1) / a.head_block;
    const long long ctas = (long long)rows * s.kv_heads * a.head_blocks;
    int splits = 1;
    while (splits < BA_MAX_SPLITS && ctas * splits < 296 && reach >= 64 * splits) splits *= 2;
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

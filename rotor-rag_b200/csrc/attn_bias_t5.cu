// The attention of attn_bias.cu for prompts, bf16, on the fifth-generation tensor cores:
//   score(i, j) = (q_i . k_j) scale - slope_h (i - j),   j <= i, j in i's chunk, i - j < window,
// a sink per head in the softmax's denominator, and the sigmoid of a gate on each head's output.  Keys and
// values lie in the caches, or (expanded latent attention) in rows made per head from the latents, with
// further key columns that all heads share (template parameter DR) coming from the latent cache itself.
//
// CTA: 128 query rows of one KV head (row = position x query head of the group); keys 128 at a time
// from the first key its first position sees up to its last position, so that keys outside every row's
// chunk or window are never read.  K and V tiles arrive by TMA straight from the caches
// (heads narrower than the 64 / 128 columns of a tile are zero filled).  Both products are
// tcgen05.mma.kind::f16 with float32 accumulators in tensor memory, scores double buffered:
//   S = Q K^T : A = Q from shared memory (staged once), B = K tile, head dimension contiguous
//   O_j = P V : A = P from tensor memory (written over the S buffer it came from), B = V tile as it lies
//               in the cache (value dimension contiguous: the descriptor's MN-major form, no transpose)
// Warps 0-7: two threads per query row (keys [0, 64) and [64, 128) of a tile, and the matching halves of
// the output columns): scale, distance bias and mask in float32, row maximum (halves exchanged through
// shared memory), exponentials (base 2), the running output O = O * alpha + O_j in registers, one tile
// behind the scores.  Warps 8 and 9: TMA of K and V; warp 10: MMA issue, one tile ahead with S.
// Waits are bounded; a wait that runs out records a code in the library status word, the CTA stops
// issuing work, frees its tensor memory and returns.  No multicast, this GPU's memory only.
#include <cstdlib>

#include "decoder.cuh"
#include "tc5.cuh"

namespace rb {

constexpr int B5_BM = 128, B5_BN = 128, B5_THREADS = 352, B5_SOFT = 256;

template <int DK, int DV, int DR>
struct B5Cfg {
    static constexpr int DQ = DK + DR;  // columns of a score
    static constexpr int Q_BYTES = B5_BM * DQ * 2, K_BYTES = B5_BN * DQ * 2, V_BYTES = B5_BN * DV * 2;
    static constexpr int RINGS = 2 * (K_BYTES + V_BYTES), BLOCKS = 8 * (int)T5_XPOSE_BYTES;  // (the output rows' blocks lie over the rings)
    static constexpr int SMEM = Q_BYTES + (RINGS > BLOCKS ? RINGS : BLOCKS) + 1024;
};

struct B5Params {
    const __nv_bfloat16* q;
    __nv_bfloat16* out;
    const int* past_len;
    const float* slopes;
    const float* sinks;
    const float* gate;
    unsigned* status;
    int heads, kv_heads, kd, vdim, ld_out, seq, max_seq, chunk, window, ld_gate;
    int rd;                          // shared key columns of a query row, behind its kd own ones
    // key j of KV head h in sequence b: row (b row_heads + h % row_heads) row_span + j - key0 of the K and V maps, from
    // columns h kx_step and vx0 + h vx_step on; its shared columns: row b max_seq + j, from column rx on
    int row_heads, row_span, key0, kx_step, vx0, vx_step, rx;
    float scale2;
};

__device__ __forceinline__ float b5_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <int DK, int DV, int DR>
__global__ void __launch_bounds__(B5_THREADS, 1)
attn_bias_t5_kernel(const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ CUtensorMap tm_r,
                    const __grid_constant__ B5Params p) {
    using C = B5Cfg<DK, DV, DR>;
    constexpr int DQ = C::DQ;
    extern __shared__ unsigned char b5_raw[];
    __shared__ __align__(8) unsigned long long s_kfull[2], s_kempty[2], s_vfull[2], s_vempty[2], s_sfull[2], s_pfull[2], s_ofull[2],
        s_oempty[2], s_qready;
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort, s_go;
    __shared__ float s_xch[2][B5_BM];
    const uint32_t qbase = (smem_u32(b5_raw) + 1023u) & ~1023u, kring = qbase + C::Q_BYTES, vring = kring + 2 * C::K_BYTES;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int G = p.heads / p.kv_heads, QT = B5_BM / G;
    const int qt = gridDim.x - 1 - blockIdx.x;  // late query tiles tend to see more keys: start them first
    const int hk = blockIdx.y, b = blockIdx.z, s0 = qt * QT;
    const int past = cached_len(p.past_len, b, p.max_seq);
    volatile int* abort_flag = &s_abort;
    const int s_last = min(s0 + QT, p.seq) - 1;
    const int p0 = past + s0;
    const int kb0 = first_visible(p0, p.chunk, p.window);
    const int t_end = min(past + s_last + 1, p.max_seq);
    const int ntiles = (t_end - kb0 + B5_BN - 1) / B5_BN;
    const int head_row = (b * p.row_heads + (p.row_heads > 1 ? hk : 0)) * p.row_span - p.key0;

    if (threadIdx.x == 0) {
        s_abort = 0;
        for (int s = 0; s < 2; ++s) {
            t5_bar_init(smem_u32(&s_kfull[s]), 1);
            t5_bar_init(smem_u32(&s_kempty[s]), 1);
            t5_bar_init(smem_u32(&s_vfull[s]), 1);
            t5_bar_init(smem_u32(&s_vempty[s]), 1);
            t5_bar_init(smem_u32(&s_sfull[s]), 1);
            t5_bar_init(smem_u32(&s_pfull[s]), B5_SOFT);
            t5_bar_init(smem_u32(&s_ofull[s]), 1);
            t5_bar_init(smem_u32(&s_oempty[s]), B5_SOFT);
        }
        t5_bar_init(smem_u32(&s_qready), B5_SOFT);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 8) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(512));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = s_tmem;  // S even [0,128)  S odd [128,256)  O even [256, +DV)  O odd [384, +DV)

    if (warp < 8) {
        {   // ---------------- Q tile, K-major panels of 64 columns, 128-byte swizzle
            constexpr int QN = B5_BM * (DQ / 8) / B5_SOFT;
            const int qd = p.kd + p.rd;
            uint4 qv[QN];
#pragma unroll
            for (int u = 0; u < QN; ++u) {
                const int idx = threadIdx.x + u * B5_SOFT, r = idx / (DQ / 8), c8 = idx - r * (DQ / 8);
                const int sp = r / G, s = s0 + sp, gi = r - sp * G;
                // own key columns, then the shared ones; what lies between in a panel is zero
                const int col = c8 < DK / 8 ? c8 * 8 : p.kd + c8 * 8 - DK;
                const bool on = c8 < DK / 8 ? col < p.kd : col < qd;
                qv[u] = make_uint4(0u, 0u, 0u, 0u);
                if (sp < QT && s < p.seq && on)
                    qv[u] = __ldg(reinterpret_cast<const uint4*>(p.q + (((size_t)b * p.seq + s) * p.heads + hk * G + gi) * qd + col));
            }
#pragma unroll
            for (int u = 0; u < QN; ++u) {
                const int idx = threadIdx.x + u * B5_SOFT, r = idx / (DQ / 8), c8 = idx - r * (DQ / 8);
                const uint32_t dst = qbase + (uint32_t)(c8 >> 3) * 16384u + (uint32_t)(r >> 3) * 1024u + (uint32_t)(r & 7) * 128u +
                                     (uint32_t)(((c8 & 7) ^ (r & 7)) << 4);
                asm volatile("st.shared.v4.u32 [%0], {%1, %2, %3, %4};" ::"r"(dst), "r"(qv[u].x), "r"(qv[u].y), "r"(qv[u].z), "r"(qv[u].w)
                             : "memory");
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");  // generic writes -> tensor-core reads
            t5_bar_arrive(smem_u32(&s_qready));
        }
        constexpr int DH = DV / 2;  // output columns of this thread
        const int half = warp >> 2, wq = warp & 3, r = wq * 32 + lane;
        const int sp = min(r / G, QT - 1), gi = r - (r / G) * G;
        const int pos = past + min(s0 + sp, s_last);
        const int lo = first_visible(pos, p.chunk, p.window), hi = pos;  // visible keys [lo, hi]
        const float slope2 = p.slopes ? __ldg(p.slopes + hk * G + gi) * 1.4426950408889634f : 0.f;
        const uint32_t lane_base = tmem + ((uint32_t)(wq * 32) << 16);
        float m_run = -INFINITY, l_run = 0.f, alpha_prev = 1.f;
        float o[DH];
#pragma unroll
        for (int i = 0; i < DH; ++i) o[i] = 0.f;
        bool ok = true;
        auto accumulate = [&](int j, float alpha) {
            const bool good = t5_wait(smem_u32(&s_ofull[j & 1]), (uint32_t)(j >> 1) & 1u, abort_flag, p.status, 0x79000002u);
            if (!__all_sync(0xffffffffu, good)) return false;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const uint32_t ob = lane_base + 256u + (uint32_t)(j & 1) * 128u + (uint32_t)half * DH;
#pragma unroll
            for (int c = 0; c < DH; c += 32) {
                uint32_t v[32];
                t5_ld32(ob + c, v);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                for (int i = 0; i < 32; ++i) o[c + i] = o[c + i] * alpha + __uint_as_float(v[i]);
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            t5_bar_arrive(smem_u32(&s_oempty[j & 1]));
            return true;
        };
        // (the eight warps leave this loop together: whether to go on is decided by one thread between the
        // two barriers of an iteration, so that no warp is left alone at a barrier after a failed wait)
        for (int j = 0; j < ntiles; ++j) {
            const uint32_t sbuf = lane_base + (uint32_t)(j & 1) * 128u;
            ok = ok && t5_wait(smem_u32(&s_sfull[j & 1]), (uint32_t)(j >> 1) & 1u, abort_flag, p.status, 0x79000001u);
            ok = __all_sync(0xffffffffu, ok);
            float sa[64];
            float tmax = -INFINITY;
            if (ok) {
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const int kb = kb0 + j * B5_BN + half * 64;
                const float base = slope2 * (float)(kb - pos);
#pragma unroll
                for (int c = 0; c < 64; c += 32) {
                    uint32_t v[32];
                    t5_ld32(sbuf + (uint32_t)half * 64u + c, v);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int i = 0; i < 32; ++i) sa[c + i] = __uint_as_float(v[i]) * p.scale2 + (slope2 * (float)(c + i) + base);
                }
                if (kb < lo || kb + 63 > hi) {
#pragma unroll
                    for (int c = 0; c < 64; ++c)
                        if (kb + c < lo || kb + c > hi) sa[c] = -INFINITY;
                }
#pragma unroll
                for (int c = 0; c < 64; ++c) tmax = fmaxf(tmax, sa[c]);
            }
            // the two threads of a row exchange their maxima; past this barrier both have finished reading the S
            // buffer, which the P stores below overwrite (every softmax warp takes part, also after a failed wait)
            s_xch[half][r] = tmax;
            asm volatile("bar.sync 1, %0;" ::"n"(B5_SOFT) : "memory");
            tmax = fmaxf(tmax, s_xch[half ^ 1][r]);
            if (threadIdx.x == 0) s_go = !*abort_flag;
            asm volatile("bar.sync 1, %0;" ::"n"(B5_SOFT) : "memory");  // the exchange slots are free again
            if (!s_go) {
                ok = false;
                break;
            }
            const float m_new = fmaxf(m_run, tmax);
            const float m_sub = m_new == -INFINITY ? 0.f : m_new;  // (no key of this row yet: an earlier chunk's tile)
            const float alpha = b5_exp2(m_run - m_sub);
            float sum = 0.f;
            uint32_t pk[32];
#pragma unroll
            for (int c = 0; c < 32; ++c) {
                const float e0 = b5_exp2(sa[2 * c] - m_sub), e1 = b5_exp2(sa[2 * c + 1] - m_sub);
                sum += e0 + e1;
                pk[c] = t5_pack(e0, e1);
            }
            t5_st32(sbuf + (uint32_t)half * 32u, pk);  // 128 bf16 weights in columns [0, 64) of the S buffer
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            t5_bar_arrive(smem_u32(&s_pfull[j & 1]));
            l_run = l_run * alpha + sum;
            m_run = m_new;
            if (j > 0) ok = accumulate(j - 1, alpha_prev);
            alpha_prev = alpha;
        }
        if (ok && ntiles > 0) ok = accumulate(ntiles - 1, alpha_prev);
        s_xch[half][r] = l_run;
        asm volatile("bar.sync 1, %0;" ::"n"(B5_SOFT) : "memory");
        l_run += s_xch[half ^ 1][r];
        if (__all_sync(0xffffffffu, ok)) {
            // rows leave through a per-warp block of the operand rings (idle: every MMA has completed)
            float inv = 1.0f / l_run;
            if (p.sinks) {
                const float sink = __ldg(p.sinks + hk * G + gi) * 1.4426950408889634f, top = fmaxf(m_run, sink), mine = b5_exp2(m_run - top);
                inv = mine / (l_run * mine + b5_exp2(sink - top));
            }
            if (p.gate) inv *= sigmoid(__ldg(p.gate + ((size_t)b * p.seq + min(s0 + sp, s_last)) * p.ld_gate + hk * G + gi));
            const uint32_t blk = kring + (uint32_t)warp * T5_XPOSE_BYTES;
            const int cpl = lane & (DV == 128 ? 7 : 3);  // 16-byte piece this lane stores
            auto dst_of = [&](int tl) -> void* {
                const int r2 = wq * 32 + tl, sp2 = r2 / G, s2 = s0 + sp2, col = half * DH + cpl * 8;
                if (sp2 >= QT || s2 >= p.seq || col >= p.vdim) return nullptr;
                return p.out + ((size_t)b * p.seq + s2) * p.ld_out + (size_t)(hk * G + r2 - sp2 * G) * p.vdim + half * DH;
            };
            if constexpr (DV == 128) {
                uint32_t v[32];
#pragma unroll
                for (int i = 0; i < 32; ++i) v[i] = t5_pack(o[2 * i] * inv, o[2 * i + 1] * inv);
                t5_store_rows_to(blk, v, lane, dst_of);
            } else {
                uint32_t v[16];
#pragma unroll
                for (int i = 0; i < 16; ++i) v[i] = t5_pack(o[2 * i] * inv, o[2 * i + 1] * inv);
                t5_store_half_rows_to(blk, v, lane, dst_of);
            }
        }
    } else if (warp == 8) {
        if (lane == 0) {
            for (int j = 0; j < ntiles; ++j) {
                const int s = j & 1;
                if (!t5_wait(smem_u32(&s_kempty[s]), ((uint32_t)(j >> 1) & 1u) ^ 1u, abort_flag, p.status, 0x79000003u)) break;
                const uint32_t bar = smem_u32(&s_kfull[s]);
                t5_bar_expect(bar, C::K_BYTES);
#pragma unroll
                for (int pn = 0; pn < DK / 64; ++pn)
                    t5_tma_2d(kring + s * C::K_BYTES + pn * 16384, &tm_k, hk * p.kx_step + pn * 64, head_row + kb0 + j * B5_BN, bar);
                if constexpr (DR > 0)
                    t5_tma_2d(kring + s * C::K_BYTES + (DK / 64) * 16384, &tm_r, p.rx, b * p.max_seq + kb0 + j * B5_BN, bar);
            }
        }
    } else if (warp == 9) {
        if (lane == 0) {
            for (int j = 0; j < ntiles; ++j) {
                const int s = j & 1;
                if (!t5_wait(smem_u32(&s_vempty[s]), ((uint32_t)(j >> 1) & 1u) ^ 1u, abort_flag, p.status, 0x79000009u)) break;
                const uint32_t bar = smem_u32(&s_vfull[s]);
                t5_bar_expect(bar, C::V_BYTES);
#pragma unroll
                for (int pn = 0; pn < DV / 64; ++pn)
                    t5_tma_2d(vring + s * C::V_BYTES + pn * 16384, &tm_v, p.vx0 + hk * p.vx_step + pn * 64, head_row + kb0 + j * B5_BN, bar);
            }
        }
    } else {
        if (lane == 0) {
            constexpr uint32_t idesc_s = t5_idesc_bf16(128, B5_BN), idesc_o = t5_idesc_bf16(128, DV, true);
            const uint64_t dq = t5_desc(qbase);
            auto issue_s = [&](int j) {
                const uint64_t dk = t5_desc(kring + (uint32_t)(j & 1) * C::K_BYTES);
#pragma unroll
                for (int k16 = 0; k16 < DQ / 16; ++k16) {
                    const uint64_t off = (uint64_t)(((k16 >> 2) * 16384 + (k16 & 3) * 32) >> 4);
                    t5_mma_ss(tmem + (uint32_t)(j & 1) * 128u, dq + off, dk + off, idesc_s, k16 > 0);
                }
                t5_commit(smem_u32(&s_sfull[j & 1]));
                t5_commit(smem_u32(&s_kempty[j & 1]));
            };
            auto issue_pv = [&](int j) {
                const uint64_t dv = t5_desc_mn(vring + (uint32_t)(j & 1) * C::V_BYTES, 16384);
#pragma unroll
                for (int k16 = 0; k16 < B5_BN / 16; ++k16)
                    t5_mma_ts(tmem + 256u + (uint32_t)(j & 1) * 128u, tmem + (uint32_t)(j & 1) * 128u + (uint32_t)k16 * 8u,
                              dv + (uint64_t)(k16 * 2048 >> 4), idesc_o, k16 > 0);
                t5_commit(smem_u32(&s_ofull[j & 1]));
                t5_commit(smem_u32(&s_vempty[j & 1]));
            };
            bool ok = t5_wait(smem_u32(&s_qready), 0, abort_flag, p.status, 0x79000004u);
            if (ok && ntiles > 0) {
                ok = t5_wait(smem_u32(&s_kfull[0]), 0, abort_flag, p.status, 0x79000005u);
                if (ok) {
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    issue_s(0);
                }
            }
            for (int j = 0; j < ntiles && ok; ++j) {
                if (j + 1 < ntiles) {
                    ok = t5_wait(smem_u32(&s_kfull[(j + 1) & 1]), (uint32_t)((j + 1) >> 1) & 1u, abort_flag, p.status, 0x79000006u);
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    issue_s(j + 1);
                }
                ok = t5_wait(smem_u32(&s_pfull[j & 1]), (uint32_t)(j >> 1) & 1u, abort_flag, p.status, 0x79000007u);
                if (ok) ok = t5_wait(smem_u32(&s_oempty[j & 1]), ((uint32_t)(j >> 1) & 1u) ^ 1u, abort_flag, p.status, 0x79000008u);
                if (ok) ok = t5_wait(smem_u32(&s_vfull[j & 1]), (uint32_t)(j >> 1) & 1u, abort_flag, p.status, 0x7900000au);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                issue_pv(j);
            }
        }
    }

    // ---------------- common exit: nothing of this CTA may still be in flight when it returns
    if (*abort_flag && threadIdx.x == 0) {
        const long long t0 = clock64();
        while (clock64() - t0 < 2000000LL) {
        }  // about a millisecond for copies already issued to land
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 8) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512));
    }
}

bool bias_attn_t5_supported(const BiasAttn& p, int rows) {
    static const bool off = getenv("ROTOR_B200_NO_TCGEN05") != nullptr;  // comparison aid: the row kernel
    const HeadShape& s = p.s;
    const int G = s.heads / s.kv_heads;
    return !off && !p.f32 && p.q && p.cache.seq >= 16 && rows % p.cache.seq == 0 && s.dim <= 128 && s.vdim <= 128 && s.vdim % 8 == 0 &&
           G <= B5_BM && p.ld_out % 8 == 0 && ((uintptr_t)p.out & 15) == 0 && s.kv_heads <= 65535 && rows / p.cache.seq <= 65535;
}

template <int DK, int DV, int DR>
static int b5_go(const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& tr, B5Params& a, int batch, cudaStream_t st) {
    using C = B5Cfg<DK, DV, DR>;
    static PerDevice<bool> once;
    if (!once.here()) {
        RB_CUDA(cudaFuncSetAttribute(attn_bias_t5_kernel<DK, DV, DR>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM));
        once.here() = true;
    }
    a.status = library_status_word();
    if (!a.status) return ROTOR_B200_ERR_CUDA;
    const int QT = B5_BM / (a.heads / a.kv_heads);
    dim3 grid((a.seq + QT - 1) / QT, a.kv_heads, batch);
    attn_bias_t5_kernel<DK, DV, DR><<<grid, B5_THREADS, C::SMEM, st>>>(tk, tv, tr, a);
    return launch_status();
}

int launch_bias_attn_t5(const BiasAttn& p, int rows, cudaStream_t st) {
    if (!bias_attn_t5_supported(p, rows)) return ROTOR_B200_ERR_SHAPE;
    const HeadShape& s = p.s;
    const int batch = rows / p.cache.seq;
    const size_t crows = (size_t)batch * s.kv_heads * p.cache.max_seq;
    if (crows > 0x7fffffffu) return ROTOR_B200_ERR_SHAPE;
    CUtensorMap tk, tv;
    if (!t5_map_bf16(&tk, p.cache.k, crows, s.kd, s.kd, B5_BN) || !t5_map_bf16(&tv, p.cache.v, crows, s.vd, s.vd, B5_BN))
        return ROTOR_B200_ERR_CUDA;
    B5Params a = {};
    a.q = p.q;
    a.out = static_cast<__nv_bfloat16*>(p.out);
    a.past_len = p.cache.past_len;
    a.slopes = p.slopes;
    a.sinks = p.sinks;
    a.heads = s.heads;
    a.kv_heads = s.kv_heads;
    a.kd = s.kd;
    a.vdim = s.vdim;
    a.ld_out = p.ld_out;
    a.seq = p.cache.seq;
    a.max_seq = p.cache.max_seq;
    a.chunk = p.chunk;
    a.window = p.window;
    a.row_heads = s.kv_heads;
    a.row_span = p.cache.max_seq;
    a.scale2 = p.scale * 1.4426950408889634f;
    const bool k64 = p.s.dim <= 64, v64 = p.s.vdim <= 64;
    if (k64) return v64 ? b5_go<64, 64, 0>(tk, tv, tk, a, batch, st) : b5_go<64, 128, 0>(tk, tv, tk, a, batch, st);
    return v64 ? b5_go<128, 64, 0>(tk, tv, tk, a, batch, st) : b5_go<128, 128, 0>(tk, tv, tk, a, batch, st);
}

bool expanded_attn_supported(const LatentShape& s, int seq) {
    static const bool off = getenv("ROTOR_B200_NO_TCGEN05") != nullptr;
    return !off && seq >= 16 && s.dp <= 128 && s.rp <= 64 && s.vdim <= 128 && s.heads <= 65535;
}

int launch_expanded_attn(const ExpandedAttn& p, int batch, cudaStream_t st) {
    const LatentShape& s = p.s;
    const int vp = (s.vdim + 7) / 8 * 8, W = latent_row(s), ld = s.heads * (s.dp + vp);
    if (!expanded_attn_supported(s, p.cache.seq)) return ROTOR_B200_ERR_SHAPE;
    RB_REQUIRE(p.q && p.kv && p.out && p.cache.rows && p.cache.past_len && batch > 0 && batch <= 65535 && p.first >= 0 && p.len > 0);
    RB_REQUIRE(p.ld_out % 8 == 0 && ((uintptr_t)p.out & 15) == 0 && (size_t)batch * p.cache.max_seq <= 0x7fffffffu);
    CUtensorMap tk, tr;
    if (!t5_map_bf16(&tk, p.kv, (size_t)batch * p.len, ld, ld, B5_BN) ||
        !t5_map_bf16(&tr, p.cache.rows, (size_t)batch * p.cache.max_seq, W, W, B5_BN))
        return ROTOR_B200_ERR_CUDA;
    B5Params a = {};
    a.q = p.q;
    a.out = p.out;
    a.past_len = p.cache.past_len;
    a.sinks = p.sinks;
    a.gate = p.gate;
    a.ld_gate = p.ld_gate;
    a.heads = a.kv_heads = s.heads;
    a.kd = s.dp;
    a.rd = s.rp;
    a.vdim = vp;
    a.ld_out = p.ld_out;
    a.seq = p.cache.seq;
    a.max_seq = p.cache.max_seq;
    a.window = p.window;
    a.row_heads = 1;
    a.row_span = p.len;
    a.key0 = p.first;
    a.kx_step = s.dp;
    a.vx0 = s.heads * s.dp;
    a.vx_step = vp;
    a.rx = s.kp;
    a.scale2 = p.scale * 1.4426950408889634f;
    const bool k64 = s.dp <= 64, v64 = vp <= 64;
    if (k64) return v64 ? b5_go<64, 64, 64>(tk, tk, tr, a, batch, st) : b5_go<64, 128, 64>(tk, tk, tr, a, batch, st);
    return v64 ? b5_go<128, 64, 64>(tk, tk, tr, a, batch, st) : b5_go<128, 128, 64>(tk, tk, tr, a, batch, st);
}

}  // namespace rb

// Dense products of many rows (prompts, batches): y = x W^T with bf16 weights.
//
// dense_gemm_t5_kernel: bf16 activations on the fifth-generation tensor cores.  Persistent CTAs, one
// per SM; a tile is 128 tokens x BN weight rows, K walked 64 at a time through a ring of TMA-loaded
// operand stages (128-byte swizzle); one thread issues tcgen05.mma.kind::f16 (M 128, N BN, K 16) into
// one of two tensor-memory accumulators, so that four read-back warps empty one tile while the next
// is computed.  BN is 256, or 64 or 32 where larger tiles would leave SMs idle.  Read-back (lane =
// token, 32 outputs per load), rows leave through a per-warp shared-memory block as whole pieces:
//   PLAIN  float32
//   GATED  a tile holds BN/2 gate rows and the matching up rows; gelu_tanh(gate) * up as bf16
//   QKV    the heads of the stacked q/k/v matrix: q and k divided by their root mean square, q rows
//          out, k and v rows to the cache positions of their tokens
// Waits are bounded; a wait that runs out records a code in the library status word, the CTA stops
// issuing work, frees its tensor memory and returns.  No multicast, this GPU's memory only.
//
// dense_gemm_f32_kernel: float32 activations on the FP32 pipe (nothing below float32 but the weights).
#include "decoder.cuh"
#include "tc5.cuh"

namespace rb {

template <int BN>
struct DgT5 {
    static constexpr int A_BYTES = 128 * 128, B_BYTES = BN * 128, STAGE = A_BYTES + B_BYTES;
    static constexpr int STAGES = BN == 256 ? 4 : (BN == 64 ? 8 : 9);
    static constexpr int XPOSE = 4 * (int)T5_XPOSE_BYTES;
    static constexpr int SMEM = STAGES * STAGE + XPOSE + 1024;
    static constexpr int TMEM_COLS = 2 * BN;
};
constexpr int DG5_THREADS = 192;  // TMA warp, MMA warp, four read-back warps

struct DgT5Params {
    unsigned* status;
    int rows, n, k, mt, nt;       // rows of x, outputs (channels when gated), K, tiles
    float* y;
    int ldy;
    __nv_bfloat16* a;
    int lda;
    HeadShape s;
    CacheView cache;
    __nv_bfloat16* q;
};

// gelu_tanh with the fast exponential and division (their error is far below the bf16 result's)
__device__ __forceinline__ float dg_gelu(float z) {
    const float t = -1.5957691216057308f * (z + 0.044715f * z * z * z);
    return __fdividef(z, 1.0f + __expf(fminf(t, 80.f)));
}

template <int BN, int EPI>
__global__ void __launch_bounds__(DG5_THREADS, 1)
dense_gemm_t5_kernel(const __grid_constant__ CUtensorMap tm_a, const __grid_constant__ CUtensorMap tm_b,
                     const __grid_constant__ DgT5Params p) {
    using C = DgT5<BN>;
    constexpr int ST = C::STAGES;
    constexpr int NB = EPI == DENSE_GATED ? 2 : (BN == 256 ? 2 : 1), BOX = BN / NB;  // weight boxes per stage
    constexpr int TN = EPI == DENSE_GATED ? BN / 2 : BN;                             // outputs per tile
    extern __shared__ unsigned char dg_raw[];
    __shared__ __align__(8) unsigned long long s_full[ST], s_empty[ST], s_accf[2], s_acce[2];
    __shared__ uint32_t s_tmem;
    __shared__ int s_abort;
    const uint32_t ring = (smem_u32(dg_raw) + 1023u) & ~1023u, xpose = ring + ST * C::STAGE;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    volatile int* abort_flag = &s_abort;
    const int nk = (p.k + 63) >> 6, ntiles = p.mt * p.nt;

    if (threadIdx.x == 0) {
        s_abort = 0;
        for (int s = 0; s < ST; ++s) {
            t5_bar_init(smem_u32(&s_full[s]), 1);
            t5_bar_init(smem_u32(&s_empty[s]), 1);
        }
        for (int s = 0; s < 2; ++s) {
            t5_bar_init(smem_u32(&s_accf[s]), 1);
            t5_bar_init(smem_u32(&s_acce[s]), 4);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&s_tmem)), "r"(C::TMEM_COLS));
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t tmem = s_tmem;

    // tiles in groups of 16 token tiles, token tiles fastest: the CTAs of a wave share weight tiles
    auto place = [&](int t, int& m, int& n) {
        const int group = t / (16 * p.nt), gm = min(16, p.mt - group * 16), r = t - group * 16 * p.nt;
        n = r / gm;
        m = group * 16 + (r - n * gm);
    };

    if (warp == 0) {
        if (lane == 0) {
            int it = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < ntiles && ok; t += gridDim.x) {
                int m, n;
                place(t, m, n);
                for (int kt = 0; kt < nk; ++kt, ++it) {
                    const int s = it % ST;
                    ok = t5_wait(smem_u32(&s_empty[s]), ((it / ST) & 1) ^ 1, abort_flag, p.status, 0x7a000001u);
                    if (!ok) break;
                    const uint32_t bar = smem_u32(&s_full[s]), st = ring + s * C::STAGE;
                    t5_bar_expect(bar, C::STAGE);
                    t5_tma_2d(st, &tm_a, kt * 64, m * 128, bar);
#pragma unroll
                    for (int b = 0; b < NB; ++b)
                        t5_tma_2d(st + C::A_BYTES + b * BOX * 128, &tm_b, kt * 64,
                                  EPI == DENSE_GATED ? b * p.n + n * TN : n * TN + b * BOX, bar);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = t5_idesc_bf16(128, BN);
            int it = 0, lt = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < ntiles && ok; t += gridDim.x, ++lt) {
                const int buf = lt & 1;
                ok = t5_wait(smem_u32(&s_acce[buf]), ((lt >> 1) & 1) ^ 1, abort_flag, p.status, 0x7a000002u);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const uint32_t d = tmem + (uint32_t)buf * BN;
                for (int kt = 0; kt < nk; ++kt, ++it) {
                    const int s = it % ST;
                    ok = t5_wait(smem_u32(&s_full[s]), (it / ST) & 1, abort_flag, p.status, 0x7a000003u);
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const uint64_t da = t5_desc(ring + s * C::STAGE), db = t5_desc(ring + s * C::STAGE + C::A_BYTES);
#pragma unroll
                    for (int k16 = 0; k16 < 4; ++k16)
                        t5_mma_ss(d, da + 2 * k16, db + 2 * k16, idesc, (kt > 0 || k16 > 0) ? 1u : 0u);
                    t5_commit(smem_u32(&s_empty[s]));
                }
                if (ok) t5_commit(smem_u32(&s_accf[buf]));
            }
        }
    } else {
        const int wq = warp & 3;  // the quarter of the tensor-memory lanes this warp reaches
        const uint32_t stage = xpose + (uint32_t)(warp - 2) * T5_XPOSE_BYTES;
        int lt = 0;
        for (int t = blockIdx.x; t < ntiles; t += gridDim.x, ++lt) {
            int m, n;
            place(t, m, n);
            const int buf = lt & 1;
            const bool good = t5_wait(smem_u32(&s_accf[buf]), (lt >> 1) & 1, abort_flag, p.status, 0x7a000004u);
            if (!__all_sync(0xffffffffu, good)) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int tok0 = m * 128 + wq * 32;
            const uint32_t tb = tmem + ((uint32_t)(wq * 32) << 16) + (uint32_t)buf * BN;
            if constexpr (EPI == DENSE_PLAIN) {
#pragma unroll 1
                for (int c = 0; c < BN / 32; ++c) {
                    const int col = n * TN + c * 32;
                    if (col >= p.ldy) break;  // (ldy is a multiple of 32; columns past n are zeros)
                    uint32_t v[32];
                    t5_ld32(tb + c * 32, v);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                    t5_store_rows(stage, v, p.y + (size_t)tok0 * p.ldy + col, (size_t)p.ldy * 4, tok0, p.rows, lane);
                }
            } else if constexpr (EPI == DENSE_GATED) {
#pragma unroll 1
                for (int c = 0; c < TN / 32; ++c) {
                    const int col = n * TN + c * 32;
                    if (col >= p.lda) break;
                    uint32_t g[32], u[32], o[16];
                    t5_ld32(tb + c * 32, g);
                    t5_ld32(tb + TN + c * 32, u);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int i = 0; i < 16; ++i) {
                        const float a = dg_gelu(__uint_as_float(g[2 * i])) * __uint_as_float(u[2 * i]);
                        const float b = dg_gelu(__uint_as_float(g[2 * i + 1])) * __uint_as_float(u[2 * i + 1]);
                        o[i] = t5_pack(col + 2 * i < p.n ? a : 0.f, col + 2 * i + 1 < p.n ? b : 0.f);
                    }
                    t5_store_half_rows_to(stage, o, lane, [&](int tl) -> void* {
                        return tok0 + tl < p.rows ? p.a + (size_t)(tok0 + tl) * p.lda + col : nullptr;
                    });
                }
            } else {
                const int dim = p.s.dim, dq = p.s.heads * dim, dk = p.s.kv_heads * dim;
                float inv = 1.f;
                int done = 0;  // columns of the tile below `done` belong to heads whose norm is known
#pragma unroll 1
                for (int c = 0; c < BN / 32; ++c) {
                    const int col = n * TN + c * 32;
                    if (col >= p.n) break;
                    const int kind = col < dq ? 0 : (col < dq + dk ? 1 : 2);
                    if (kind == 2) {
                        inv = 1.f;
                    } else if (c * 32 >= done) {  // a new head: its columns are all in this tile
                        inv = 1.f;
                        if (p.s.unit) {
                            float ss = 0.f;
#pragma unroll 1
                            for (int e = 0; e < dim; e += 32) {
                                uint32_t v[32];
                                t5_ld32(tb + c * 32 + e, v);
                                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                                for (int i = 0; i < 32; ++i) ss += __uint_as_float(v[i]) * __uint_as_float(v[i]);
                            }
                            inv = 1.0f / sqrtf(ss / (float)dim + p.s.eps);
                        }
                        done = c * 32 + dim;
                    }
                    uint32_t v[32], o[16];
                    t5_ld32(tb + c * 32, v);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int i = 0; i < 16; ++i)
                        o[i] = t5_pack(__uint_as_float(v[2 * i]) * inv, __uint_as_float(v[2 * i + 1]) * inv);
                    const int wide = kind == 2 ? p.s.vdim : dim, rel = kind == 0 ? col : (kind == 1 ? col - dq : col - dq - dk);
                    const int head = rel / wide, off = rel - head * wide;
                    t5_store_half_rows_to(stage, o, lane, [&](int tl) -> void* {
                        const int tok = tok0 + tl;
                        if (tok >= p.rows) return nullptr;
                        if (kind == 0) return p.q + (size_t)tok * dq + col;  // (kd == dim)
                        const int b = tok / p.cache.seq, pos = cached_len(p.cache.past_len, b, p.cache.max_seq) + (tok - b * p.cache.seq);
                        if (pos >= p.cache.max_seq) return nullptr;
                        __nv_bfloat16* base = static_cast<__nv_bfloat16*>(kind == 1 ? p.cache.k : p.cache.v);
                        return base + (((size_t)b * p.s.kv_heads + head) * p.cache.max_seq + pos) * wide + off;
                    });
                }
            }
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) t5_bar_arrive(smem_u32(&s_acce[buf]));
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
    if (warp == 0) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(C::TMEM_COLS));
    }
}

bool dense_gemm_t5_supported(const DenseProduct& p, int rows) {
    if (p.f32 || rows < 1 || p.ldw % 8 || p.ldx % 8 || ((uintptr_t)p.w & 15) || ((uintptr_t)p.x & 15)) return false;
    if (p.epilogue == DENSE_PLAIN) return p.ldy % 32 == 0;
    if (p.epilogue == DENSE_GATED) return p.lda % 32 == 0;
    // heads that never straddle a 64-column tile, cache rows without padding
    const HeadShape& s = p.shape;
    return (s.dim == 32 || s.dim == 64 || s.dim == 128) && s.vdim % 32 == 0 && s.kd == s.dim && s.vd == s.vdim;
}

template <int BN, int EPI>
static int dg5_launch(const DenseProduct& p, int rows, cudaStream_t st) {
    using C = DgT5<BN>;
    constexpr int NB = EPI == DENSE_GATED ? 2 : (BN == 256 ? 2 : 1), BOX = BN / NB, TN = EPI == DENSE_GATED ? BN / 2 : BN;
    static PerDevice<bool> once;
    if (!once.here()) {
        RB_CUDA(cudaFuncSetAttribute(dense_gemm_t5_kernel<BN, EPI>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM));
        once.here() = true;
    }
    DgT5Params a = {};
    a.status = library_status_word();
    if (!a.status) return ROTOR_B200_ERR_CUDA;
    a.rows = rows;
    a.n = p.n;
    a.k = p.k;
    a.mt = (rows + 127) / 128;
    a.nt = (p.n + TN - 1) / TN;
    a.y = p.y;
    a.ldy = p.ldy;
    a.a = static_cast<__nv_bfloat16*>(p.a);
    a.lda = p.lda;
    a.s = p.shape;
    a.cache = p.cache;
    a.q = p.q;
    CUtensorMap ta, tb;
    if (!t5_map_bf16(&ta, p.x, rows, p.k, p.ldx, 128) ||
        !t5_map_bf16(&tb, p.w, (size_t)p.n * (EPI == DENSE_GATED ? 2 : 1), p.k, p.ldw, BOX))
        return ROTOR_B200_ERR_CUDA;
    const int tiles = a.mt * a.nt, sms = fused_sm_count();
    dense_gemm_t5_kernel<BN, EPI><<<tiles < sms ? tiles : sms, DG5_THREADS, C::SMEM, st>>>(ta, tb, a);
    return launch_status();
}

int launch_dense_gemm_t5(const DenseProduct& p, int rows, cudaStream_t st) {
    if (!dense_gemm_t5_supported(p, rows)) return ROTOR_B200_ERR_SHAPE;
    const int tn = p.epilogue == DENSE_GATED ? 128 : 256;
    bool wide = (long long)((rows + 127) / 128) * ((p.n + tn - 1) / tn) >= fused_sm_count();
    if (p.epilogue == DENSE_QKV && p.shape.dim > 64) wide = true;
    switch (p.epilogue) {
        case DENSE_PLAIN:
            if (wide) return dg5_launch<256, DENSE_PLAIN>(p, rows, st);
            // (a few dozen rows of a narrow output: the weight stream wants as many CTAs as there are)
            return (long long)((rows + 127) / 128) * ((p.n + 63) / 64) * 4 >= 3LL * fused_sm_count() ? dg5_launch<64, DENSE_PLAIN>(p, rows, st)
                                                                                                   : dg5_launch<32, DENSE_PLAIN>(p, rows, st);
        case DENSE_GATED: return wide ? dg5_launch<256, DENSE_GATED>(p, rows, st) : dg5_launch<64, DENSE_GATED>(p, rows, st);
        default: return wide ? dg5_launch<256, DENSE_QKV>(p, rows, st) : dg5_launch<64, DENSE_QKV>(p, rows, st);
    }
}

// ---------------------------------------------------------------------------------------
// 64 x 64 tiles, 4 x 4 outputs per thread, K 16 at a time.
__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const float* __restrict__ x, int ldx, const __nv_bfloat16* __restrict__ w,
                                                             int ldw, int rows, int n, int k, float* __restrict__ y, int ldy) {
    __shared__ __align__(16) float xs[16][68], ws[16][68];
    const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < k; k0 += 16) {
        float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
        if (m0 + lr < rows) {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (k0 + lk + e < k) a[e] = x[(size_t)(m0 + lr) * ldx + k0 + lk + e];
        }
        if (n0 + lr < n) {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (k0 + lk + e < k) b[e] = __bfloat162float(w[(size_t)(n0 + lr) * ldw + k0 + lk + e]);
        }
        __syncthreads();
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            xs[lk + e][lr] = a[e];
            ws[lk + e][lr] = b[e];
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < 16; ++kk) {
            const float4 av = *reinterpret_cast<const float4*>(&xs[kk][ty * 4]), bv = *reinterpret_cast<const float4*>(&ws[kk][tx * 4]);
            const float am[4] = {av.x, av.y, av.z, av.w}, bm[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] += am[i] * bm[j];
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int r = m0 + ty * 4 + i;
        if (r >= rows) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (n0 + tx * 4 + j < n) y[(size_t)r * ldy + n0 + tx * 4 + j] = acc[i][j];
    }
}

__global__ void __launch_bounds__(256) gate_f32_kernel(const float* __restrict__ gu, int ldgu, int rows, int ff, float* __restrict__ a, int lda) {
    const size_t total = (size_t)rows * ff;
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < total; i += (size_t)gridDim.x * 256) {
        const int r = (int)(i / ff), c = (int)(i - (size_t)r * ff);
        a[(size_t)r * lda + c] = gelu_tanh(gu[(size_t)r * ldgu + c]) * gu[(size_t)r * ldgu + ff + c];
    }
}

// gate_up: scratch of a gated product, float32 [rows][2 n]
int launch_dense_gemm_f32(const DenseProduct& p, int rows, float* gate_up, cudaStream_t st) {
    RB_REQUIRE(p.f32 && p.w && p.x && rows > 0 && p.epilogue != DENSE_QKV);
    const bool gated = p.epilogue == DENSE_GATED;
    RB_REQUIRE(gated ? (gate_up && p.a) : p.y != nullptr);
    const int n = gated ? 2 * p.n : p.n;
    float* y = gated ? gate_up : p.y;
    const int ldy = gated ? 2 * p.n : p.ldy;
    for (int r0 = 0; r0 < rows; r0 += 65535 * 64) {
        const int m = rows - r0 < 65535 * 64 ? rows - r0 : 65535 * 64;
        dim3 grid((n + 63) / 64, (m + 63) / 64);
        dense_gemm_f32_kernel<<<grid, 256, 0, st>>>(static_cast<const float*>(p.x) + (size_t)r0 * p.ldx, p.ldx, p.w, p.ldw, m, n, p.k,
                                                    y + (size_t)r0 * ldy, ldy);
        int rc = launch_status();
        if (rc) return rc;
    }
    if (!gated) return ROTOR_B200_OK;
    const size_t total = (size_t)rows * p.n, blocks = (total + 255) / 256;
    gate_f32_kernel<<<(unsigned)(blocks < 148 * 16 ? blocks : 148 * 16), 256, 0, st>>>(gate_up, 2 * p.n, rows, p.n,
                                                                                        static_cast<float*>(p.a), p.lda);
    return launch_status();
}

int configure_dense_gemv();
int configure_dense() { return configure_dense_gemv(); }

}  // namespace rb

// Dense products of many rows (prompts, batches): y = x W^T with bf16 weights.
//
// dense_gemm_t5_kernel: bf16 activations on the fifth-generation tensor cores.  Persistent CTAs, one
// per SM; a tile is 128 tokens x BN weight rows, K walked 64 at a time through a ring of TMA-loaded
// operand stages (128-byte swizzle); one thread issues tcgen05.mma.kind::f16 (M 128, N BN, K 16) into
// one of two tensor-memory accumulators, so that four read-back warps empty one tile while the next
// is computed.  BN is 256, or 64 or 32 where larger tiles would leave SMs idle.  Read-back (lane =
// token, 32 outputs per load), rows leave through a per-warp shared-memory block as whole pieces:
//   PLAIN  float32
//   HALF   bf16, optionally times the sigmoid of a gate per token and group
//   GATED  a tile holds BN/2 gate rows and the matching up rows; act(gate) * up as bf16
//   ROPE   query heads with their rotated columns turned by the token's position as bf16 rows, what lies behind
//          them as float32
//   QKV    the heads of the stacked q/k/v matrix: q and k divided by their root mean square, q rows
//          out, k and v rows to the cache positions of their tokens
// Groups (heads, sequences, experts) are more tiles of the same launch: a tile's operand and output origins
// come from its group, or, for experts, from the table of slot runs the routing made.
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
    int act, groups, gx_col, gx_row, gw_row, gy_col, gy_row;
    const float* head_gate;
    int ld_head_gate;
    int q_cols, rot_at, rot;
    const float2* rope;
    const int* table;             // experts: tile count, then (expert, first slot, slots) per tile of tokens
};

// Origins of one tile.
struct DgTile {
    int x_row, x_col, w_row;      // operands
    int n;                        // tile of outputs
    int row0, rows;               // first output row; rows from there on that are this tile's own
    int group, y_col;
};

// gelu_tanh with the fast exponential and division (their error is far below the bf16 result's)
__device__ __forceinline__ float dg_gelu(float z) {
    const float t = -1.5957691216057308f * (z + 0.044715f * z * z * z);
    return __fdividef(z, 1.0f + __expf(fminf(t, 80.f)));
}
__device__ __forceinline__ float dg_silu(float z) { return __fdividef(z, 1.0f + __expf(fminf(-z, 80.f))); }

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
    const int nk = (p.k + 63) >> 6;
    const int mt = p.table ? __ldg(p.table) : p.mt, per_group = mt * p.nt, ntiles = per_group * p.groups;

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

    // tiles in blocks of 16 token tiles, token tiles fastest: the CTAs of a wave share weight tiles
    auto place = [&](int t) {
        DgTile o;
        o.group = t / per_group;
        t -= o.group * per_group;
        const int block = t / (16 * p.nt), bm = min(16, mt - block * 16), r = t - block * 16 * p.nt;
        o.n = r / bm;
        const int m = block * 16 + (r - o.n * bm);
        if (p.table) {
            const int* e = p.table + 1 + 3 * m;
            o.group = __ldg(e);
            o.x_row = o.row0 = __ldg(e + 1);
            o.rows = __ldg(e + 2);
            o.x_col = o.y_col = 0;
        } else {
            o.x_row = o.group * p.gx_row + m * 128;
            o.x_col = o.group * p.gx_col;
            o.row0 = o.group * p.gy_row + m * 128;
            o.rows = p.rows - m * 128;
            o.y_col = o.group * p.gy_col;
        }
        o.w_row = o.group * p.gw_row;
        return o;
    };

    if (warp == 0) {
        if (lane == 0) {
            int it = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < ntiles && ok; t += gridDim.x) {
                const DgTile at = place(t);
                for (int kt = 0; kt < nk; ++kt, ++it) {
                    const int s = it % ST;
                    ok = t5_wait(smem_u32(&s_empty[s]), ((it / ST) & 1) ^ 1, abort_flag, p.status, 0x7a000001u);
                    if (!ok) break;
                    const uint32_t bar = smem_u32(&s_full[s]), st = ring + s * C::STAGE;
                    t5_bar_expect(bar, C::STAGE);
                    t5_tma_2d(st, &tm_a, at.x_col + kt * 64, at.x_row, bar);
#pragma unroll
                    for (int b = 0; b < NB; ++b)
                        t5_tma_2d(st + C::A_BYTES + b * BOX * 128, &tm_b, kt * 64,
                                  at.w_row + (EPI == DENSE_GATED ? b * p.n + at.n * TN : at.n * TN + b * BOX), bar);
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
            const DgTile at = place(t);
            const int n = at.n;
            const int buf = lt & 1;
            const bool good = t5_wait(smem_u32(&s_accf[buf]), (lt >> 1) & 1, abort_flag, p.status, 0x7a000004u);
            if (!__all_sync(0xffffffffu, good)) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int tok0 = at.row0 + wq * 32, tok_end = at.row0 + at.rows;
            const uint32_t tb = tmem + ((uint32_t)(wq * 32) << 16) + (uint32_t)buf * BN;
            if constexpr (EPI == DENSE_PLAIN) {
#pragma unroll 1
                for (int c = 0; c < BN / 32; ++c) {
                    const int col = n * TN + c * 32;
                    if (col >= p.ldy) break;  // (ldy is a multiple of 32; columns past n are zeros)
                    uint32_t v[32];
                    t5_ld32(tb + c * 32, v);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                    t5_store_rows(stage, v, p.y + (size_t)tok0 * p.ldy + col, (size_t)p.ldy * 4, tok0, tok_end, lane);
                }
            } else if constexpr (EPI == DENSE_HALF) {
                float gate = 1.f;
                if (p.head_gate && tok0 + lane < tok_end) gate = sigmoid(__ldg(p.head_gate + (size_t)(tok0 + lane) * p.ld_head_gate + at.group));
#pragma unroll 1
                for (int c = 0; c < BN / 32; ++c) {
                    const int col = n * TN + c * 32;
                    if (col >= p.n) break;
                    uint32_t v[32], o[16];
                    t5_ld32(tb + c * 32, v);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
                    for (int i = 0; i < 16; ++i)
                        o[i] = t5_pack(col + 2 * i < p.n ? __uint_as_float(v[2 * i]) * gate : 0.f,
                                       col + 2 * i + 1 < p.n ? __uint_as_float(v[2 * i + 1]) * gate : 0.f);
                    // (groups are a multiple of eight wide: 16-byte pieces past one belong to the next)
                    const int piece = (lane & 3) * 8;
                    t5_store_half_rows_to(stage, o, lane, [&](int tl) -> void* {
                        return tok0 + tl < tok_end && col + piece < p.n ? p.a + (size_t)(tok0 + tl) * p.lda + at.y_col + col : nullptr;
                    });
                }
            } else if constexpr (EPI == DENSE_ROPE) {
                const int tok = min(tok0 + lane, p.rows - 1), b = tok / p.cache.seq;
                const int pos = min(cached_len(p.cache.past_len, b, p.cache.max_seq) + (tok - b * p.cache.seq), p.cache.max_seq - 1);
                const float2* rope = p.rope + (size_t)pos * (p.rot >> 1);
                const int qd = p.rot_at + p.rot;
#pragma unroll 1
                for (int c = 0; c < BN / 32; ++c) {
                    const int col = n * TN + c * 32;
                    if (col >= p.ldy) break;
                    uint32_t v[32];
                    t5_ld32(tb + c * 32, v);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                    if (col >= p.q_cols) {
                        t5_store_rows(stage, v, p.y + (size_t)tok0 * p.ldy + col, (size_t)p.ldy * 4, tok0, tok_end, lane);
                        continue;
                    }
                    uint32_t o[16];
                    const int turn = col % qd - p.rot_at;  // (columns of a chunk are all plain or all rotated)
                    if (turn < 0) {
#pragma unroll
                        for (int i = 0; i < 16; ++i) o[i] = t5_pack(__uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1]));
                    } else {
                        const float4* cs = reinterpret_cast<const float4*>(rope + (turn >> 1));
#pragma unroll
                        for (int i = 0; i < 8; ++i) {
                            const float4 t = __ldg(cs + i);
                            const float a = __uint_as_float(v[4 * i]), b2 = __uint_as_float(v[4 * i + 1]), e = __uint_as_float(v[4 * i + 2]),
                                        f = __uint_as_float(v[4 * i + 3]);
                            o[2 * i] = t5_pack(a * t.x - b2 * t.y, b2 * t.x + a * t.y);
                            o[2 * i + 1] = t5_pack(e * t.z - f * t.w, f * t.z + e * t.w);
                        }
                    }
                    t5_store_half_rows_to(stage, o, lane, [&](int tl) -> void* {
                        return tok0 + tl < tok_end ? p.q + (size_t)(tok0 + tl) * p.q_cols + col : nullptr;
                    });
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
                        const float g0 = __uint_as_float(g[2 * i]), g1 = __uint_as_float(g[2 * i + 1]);
                        const float a = (p.act == ACT_SILU ? dg_silu(g0) : dg_gelu(g0)) * __uint_as_float(u[2 * i]);
                        const float b = (p.act == ACT_SILU ? dg_silu(g1) : dg_gelu(g1)) * __uint_as_float(u[2 * i + 1]);
                        o[i] = t5_pack(col + 2 * i < p.n ? a : 0.f, col + 2 * i + 1 < p.n ? b : 0.f);
                    }
                    t5_store_half_rows_to(stage, o, lane, [&](int tl) -> void* {
                        return tok0 + tl < tok_end ? p.a + (size_t)(tok0 + tl) * p.lda + col : nullptr;
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
    if (p.epilogue == DENSE_ROPE)
        return p.ldy % 32 == 0 && p.rot_at % 32 == 0 && p.rot % 32 == 0 && p.rot > 0 && p.q_cols % (p.rot_at + p.rot) == 0 && !p.groups && !p.route;
    if (p.epilogue == DENSE_HALF) return p.lda % 8 == 0 && (!p.groups || p.n % 8 == 0) && p.gy_col % 8 == 0 && p.gx_col % 8 == 0;
    // heads that never straddle a 64-column tile, cache rows without padding
    const HeadShape& s = p.shape;
    return (s.dim == 32 || s.dim == 64 || s.dim == 128) && s.vdim % 32 == 0 && s.kd == s.dim && s.vd == s.vdim;
}

// Tokens of all groups (of a token's choices) that tiles of 128 have to cover: tile count, at most.
static long long dg5_token_tiles(const DenseProduct& p, int rows) {
    if (p.route) return route_tiles((long long)rows, p.route->experts, 128);
    return (long long)((rows + 127) / 128) * (p.groups ? p.groups : 1);
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
    const int groups = p.groups ? p.groups : 1, wn = p.n * (EPI == DENSE_GATED ? 2 : 1);
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
    a.act = p.act;
    a.groups = p.route ? 1 : groups;
    a.gx_col = p.gx_col;
    a.gx_row = p.gx_row;
    a.gw_row = p.route ? wn : p.gw_row;
    a.gy_col = p.gy_col;
    a.gy_row = p.gy_row;
    a.head_gate = p.head_gate;
    a.ld_head_gate = p.ld_head_gate;
    a.q_cols = p.q_cols;
    a.rot_at = p.rot_at;
    a.rot = p.rot;
    a.rope = p.rope;
    a.table = p.route ? p.route->table : nullptr;
    // extents of the operands, all groups together
    const size_t x_rows = (size_t)rows + (size_t)(groups - 1) * p.gx_row, x_cols = (size_t)p.k + (size_t)(groups - 1) * p.gx_col;
    const size_t w_rows = p.route ? (size_t)p.route->experts * wn : (size_t)wn + (size_t)(groups - 1) * p.gw_row;
    CUtensorMap ta, tb;
    if (!t5_map_bf16(&ta, p.x, x_rows, x_cols, p.ldx, 128) || !t5_map_bf16(&tb, p.w, w_rows, p.k, p.ldw, BOX)) return ROTOR_B200_ERR_CUDA;
    const long long tiles = dg5_token_tiles(p, rows) * a.nt;
    const int sms = fused_sm_count();
    dense_gemm_t5_kernel<BN, EPI><<<(int)(tiles < sms ? tiles : sms), DG5_THREADS, C::SMEM, st>>>(ta, tb, a);
    return launch_status();
}

int launch_dense_gemm_t5(const DenseProduct& p, int rows, cudaStream_t st) {
    if (!dense_gemm_t5_supported(p, rows)) return ROTOR_B200_ERR_SHAPE;
    RB_REQUIRE(!p.route || (p.route->table && p.route->tile_rows == 128));
    const int tn = p.epilogue == DENSE_GATED ? 128 : 256;
    const long long mt = dg5_token_tiles(p, rows);
    bool wide = mt * ((p.n + tn - 1) / tn) >= fused_sm_count();
    if (p.epilogue == DENSE_QKV && p.shape.dim > 64) wide = true;
    // (a few dozen rows of a narrow output: the weight stream wants as many CTAs as there are)
    const bool narrow = mt * ((p.n + 63) / 64) * 4 < 3LL * fused_sm_count();
    switch (p.epilogue) {
        case DENSE_PLAIN:
            if (wide) return dg5_launch<256, DENSE_PLAIN>(p, rows, st);
            return narrow ? dg5_launch<32, DENSE_PLAIN>(p, rows, st) : dg5_launch<64, DENSE_PLAIN>(p, rows, st);
        case DENSE_HALF:
            if (wide) return dg5_launch<256, DENSE_HALF>(p, rows, st);
            return narrow ? dg5_launch<32, DENSE_HALF>(p, rows, st) : dg5_launch<64, DENSE_HALF>(p, rows, st);
        case DENSE_ROPE:
            if (wide) return dg5_launch<256, DENSE_ROPE>(p, rows, st);
            return narrow ? dg5_launch<32, DENSE_ROPE>(p, rows, st) : dg5_launch<64, DENSE_ROPE>(p, rows, st);
        case DENSE_GATED: return wide ? dg5_launch<256, DENSE_GATED>(p, rows, st) : dg5_launch<64, DENSE_GATED>(p, rows, st);
        default: return wide ? dg5_launch<256, DENSE_QKV>(p, rows, st) : dg5_launch<64, DENSE_QKV>(p, rows, st);
    }
}

// ---------------------------------------------------------------------------------------
// 64 x 64 tiles, 4 x 4 outputs per thread, K 16 at a time; grid.z: groups (experts: token tiles on grid.y, from
// the table).
struct DgF32 {
    const float* x;
    const __nv_bfloat16* w;
    float* y;
    int ldx, ldw, rows, n, k, ldy;
    int gx_col, gx_row, gw_row, gy_col, gy_row;
    const float* head_gate;
    int ld_head_gate;
    const int* table;
};
__global__ void __launch_bounds__(256) dense_gemm_f32_kernel(const __grid_constant__ DgF32 p) {
    __shared__ __align__(16) float xs[16][68], ws[16][68];
    int group = blockIdx.z, m0 = blockIdx.y * 64, end = p.rows;
    if (p.table) {
        if ((int)blockIdx.y >= p.table[0]) return;
        const int* e = p.table + 1 + 3 * blockIdx.y;
        group = e[0];
        m0 = e[1];
        end = m0 + e[2];
    }
    const float* x = p.x + (size_t)group * p.gx_row * p.ldx + (size_t)group * p.gx_col;
    const __nv_bfloat16* w = p.w + (size_t)group * p.gw_row * p.ldw;
    float* y = p.y + (size_t)group * p.gy_row * p.ldy + (size_t)group * p.gy_col;
    const int n0 = blockIdx.x * 64;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.k; k0 += 16) {
        float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
        if (m0 + lr < end) {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (k0 + lk + e < p.k) a[e] = x[(size_t)(m0 + lr) * p.ldx + k0 + lk + e];
        }
        if (n0 + lr < p.n) {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (k0 + lk + e < p.k) b[e] = __bfloat162float(w[(size_t)(n0 + lr) * p.ldw + k0 + lk + e]);
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
        if (r >= end) continue;
        const float gate = p.head_gate ? sigmoid(p.head_gate[(size_t)r * p.ld_head_gate + group]) : 1.f;
#pragma unroll
        for (int j = 0; j < 4; ++j)
            if (n0 + tx * 4 + j < p.n) y[(size_t)r * p.ldy + n0 + tx * 4 + j] = acc[i][j] * gate;
    }
}

__global__ void __launch_bounds__(256) gate_f32_kernel(const float* __restrict__ gu, int ldgu, int rows, int ff, int act, float* __restrict__ a, int lda) {
    const size_t total = (size_t)rows * ff;
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < total; i += (size_t)gridDim.x * 256) {
        const int r = (int)(i / ff), c = (int)(i - (size_t)r * ff);
        a[(size_t)r * lda + c] = gate_act(act, gu[(size_t)r * ldgu + c]) * gu[(size_t)r * ldgu + ff + c];
    }
}

// gate_up: scratch of a gated product, float32 [rows][2 n]
int launch_dense_gemm_f32(const DenseProduct& p, int rows, float* gate_up, cudaStream_t st) {
    RB_REQUIRE(p.f32 && p.w && p.x && rows > 0 && p.epilogue != DENSE_QKV && p.epilogue != DENSE_ROPE);
    const bool gated = p.epilogue == DENSE_GATED;
    const int groups = p.groups ? p.groups : 1;
    RB_REQUIRE(gated ? (gate_up && p.a) : (p.epilogue == DENSE_HALF ? p.a != nullptr : p.y != nullptr));
    RB_REQUIRE(!p.route || (p.route->table && p.route->tile_rows == 64));
    RB_REQUIRE(groups <= 65535);
    DgF32 a = {};
    a.x = static_cast<const float*>(p.x);
    a.w = p.w;
    a.ldx = p.ldx;
    a.ldw = p.ldw;
    a.n = gated ? 2 * p.n : p.n;
    a.k = p.k;
    a.y = gated ? gate_up : p.epilogue == DENSE_HALF ? static_cast<float*>(p.a) : p.y;
    a.ldy = gated ? 2 * p.n : p.epilogue == DENSE_HALF ? p.lda : p.ldy;
    a.gx_col = p.gx_col;
    a.gx_row = p.gx_row;
    a.gw_row = p.route ? a.n : p.gw_row;
    a.gy_col = p.gy_col;
    a.gy_row = p.gy_row;
    a.head_gate = p.head_gate;
    a.ld_head_gate = p.ld_head_gate;
    const int limit = p.route ? rows : 65535 * 64;
    for (int r0 = 0; r0 < rows; r0 += limit) {
        const int m = rows - r0 < limit ? rows - r0 : limit;
        const int mt = p.route ? route_tiles(m, p.route->experts, 64) : (m + 63) / 64;
        RB_REQUIRE(mt <= 65535);
        DgF32 b = a;
        b.x += (size_t)r0 * p.ldx;
        b.y += (size_t)r0 * a.ldy;
        if (b.head_gate) b.head_gate += (size_t)r0 * p.ld_head_gate;
        b.rows = m;
        b.table = p.route ? p.route->table : nullptr;
        dim3 grid((a.n + 63) / 64, mt, p.route ? 1 : groups);
        dense_gemm_f32_kernel<<<grid, 256, 0, st>>>(b);
        int rc = launch_status();
        if (rc) return rc;
    }
    if (!gated) return ROTOR_B200_OK;
    const size_t total = (size_t)rows * p.n, blocks = (total + 255) / 256;
    gate_f32_kernel<<<(unsigned)(blocks < 148 * 16 ? blocks : 148 * 16), 256, 0, st>>>(gate_up, 2 * p.n, rows, p.n, p.act,
                                                                                        static_cast<float*>(p.a), p.lda);
    return launch_status();
}

int configure_dense_gemv();
int configure_dense() {
    static PerDevice<bool> once;
    if (once.here()) return ROTOR_B200_OK;
    const int rc = configure_dense_gemv();
    once.here() = rc == ROTOR_B200_OK;
    return rc;
}

}  // namespace rb

// Dense products of up to four rows (generation steps): y = x W^T with bf16 weights, bound by the weight
// stream, with the residual stage that produces x fused into the prologue and the gating into the end.
//
// Grid: two CTAs per SM, each owning a contiguous run of output rows (a gated product: of gate / up pairs).
// The run's work is a list of units (output row, 256 columns); the CTA's warps take equal contiguous
// shares of that list, so that rows are split across warps where that is what balances them, and the
// shares of a row are added in warp order (fixed order: repeated runs give identical bits).  A unit is
// one 128-bit weight load per lane; loads run a batch ahead of the arithmetic, and the first batches
// are requested before the programmatic-launch wait.
//
// Variants (MODE): products of two normed rows of one stage (the second a small one: a router), of float32 rows
// normed on the way, one product per group (grid.y: heads), and a token's experts -- the gated product of each (token, choice) with the
// expert's weights (grid.y; every CTA makes the choice itself from the router's outputs), and the weighted
// sum of their down products as one product whose K runs over the choices.
#include "decoder.cuh"

namespace rb {

constexpr int DG_THREADS = 512, DG_WARPS = DG_THREADS / 32, DG_CTAS = 296;
constexpr int DG_U = 4;                       // units per load batch
constexpr int DG_AHEAD = 16;                  // units requested into L2 ahead of the launch wait
constexpr size_t DG_SMEM_MAX = 200 * 1024;

struct DenseGemvArgs {
    DenseProduct p;
    StreamStage st;
    Routing route;
    int has_stage, rows, slots, max_rows;
};
enum { GV_PLAIN = 0, GV_DUAL = 1, GV_GROUPS = 2, GV_EXPERT_UP = 3, GV_EXPERT_DOWN = 4, GV_NORMED = 5 };

// Column i (a multiple of 4) of a staged row: the two halves of a lane's eight columns sit 128 floats
// apart, which makes both 128-bit reads of a unit free of bank conflicts.
__device__ __forceinline__ int dg_slot(int i) { return (i & ~255) + ((i >> 2) & 1) * 128 + ((i & 255) >> 3) * 4; }

template <int R, int S, int MODE>
__global__ void __launch_bounds__(DG_THREADS, R <= 2 ? 2 : 1) dense_gemv_kernel(const __grid_constant__ DenseGemvArgs a) {
    const DenseProduct& p = a.p;
    extern __shared__ __align__(16) float sm[];
    __shared__ float coef[STREAMS_MAX * STREAMS_MAX + 2 * STREAMS_MAX], red[64];
    __shared__ int s_sel[EXPERT_TOP_MAX];
    __shared__ float s_weight[EXPERT_TOP_MAX];
    constexpr bool EXPERT = MODE == GV_EXPERT_UP || MODE == GV_EXPERT_DOWN;
    const int kx = (p.k + 255) & ~255, segs = MODE == GV_EXPERT_DOWN ? a.route.top : 1, ksteps = kx >> 8, steps = ksteps * segs;
    float* xs = sm;                 // [R][kx]; two normed rows: [2][R][kx]; several experts: [top][kx]
    float* part = sm + (MODE == GV_DUAL ? 2 * R : R * segs) * kx;  // [local row][slot][R]
    const int y = (int)blockIdx.y;  // group, (token, choice), token
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool gated = p.epilogue == DENSE_GATED;
    const int n_all = MODE == GV_DUAL ? p.n + p.n2 : p.n;
    const int n0 = (int)((long long)blockIdx.x * n_all / gridDim.x), n1 = (int)((long long)(blockIdx.x + 1) * n_all / gridDim.x);
    const int lr = (n1 - n0) * (gated ? 2 : 1);
    const int units = lr * steps, upw = max(1, (units + DG_WARPS - 1) / DG_WARPS);
    const int u0 = min(units, warp * upw), u1 = min(units, u0 + upw);

    // load cursor, a batch ahead of the arithmetic cursor
    auto row_start = [&](int r, int seg) {
        int row = gated ? (r & 1) * p.n + n0 + (r >> 1) : n0 + r;
        const __nv_bfloat16* w = p.w;
        if constexpr (MODE == GV_DUAL)
            if (row >= p.n) {
                row -= p.n;
                w = p.w2;
            }
        size_t at = row;
        if constexpr (MODE == GV_GROUPS) at += (size_t)y * p.gw_row;
        if constexpr (MODE == GV_EXPERT_UP) at += (size_t)s_sel[y % a.route.top] * 2 * p.n;
        if constexpr (MODE == GV_EXPERT_DOWN) at += (size_t)s_sel[seg] * p.n;
        return w + at * p.ldw + lane * 8;
    };
    // the weights depend on the router's outputs; a down product's are older than the gated product in front of it
    const bool late = MODE == GV_EXPERT_UP && !a.route.early;
    if constexpr (EXPERT) {
        if (late) {
            pdl_wait();
            pdl_trigger();
        }
        const int row = MODE == GV_EXPERT_UP ? y / a.route.top : y;
        if (warp == 0) {
            int sel;
            float w;
            route_row(a.route, row, lane, sel, w);
            if (lane < a.route.top) {
                s_sel[lane] = sel;
                s_weight[lane] = w;
            }
        }
        __syncthreads();
    }
    int lrow = u0 / steps, lstep = u0 - lrow * steps, lseg = lstep / ksteps, lu = u0, lcol = ((lstep - lseg * ksteps) << 8) + lane * 8;
    const __nv_bfloat16* lp = row_start(lrow, lseg) + ((lstep - lseg * ksteps) << 8);
    auto fetch = [&](uint4 (&w)[DG_U]) {
#pragma unroll
        for (int j = 0; j < DG_U; ++j) {
            w[j] = make_uint4(0u, 0u, 0u, 0u);
            if (lu < u1 && lcol < p.ldw) w[j] = ld_stream_v4(reinterpret_cast<const uint4*>(lp));
            ++lu;
            lp += 256;
            lcol += 256;
            if (++lstep == steps) {
                lstep = 0;
                lseg = 0;
                lcol = lane * 8;
                lp = row_start(++lrow, 0);
            } else if (MODE == GV_EXPERT_DOWN && lstep == (lseg + 1) * ksteps) {
                lcol = lane * 8;
                lp = row_start(lrow, ++lseg);
            }
        }
    };
    uint4 wa[DG_U], wb[DG_U];
    fetch(wa);
    // the stream goes on during the prologue: the next units, a 128-byte line per lane, into L2
#pragma unroll
    for (int i = 0; i < DG_AHEAD / 8; ++i) {
        const int u = u0 + DG_U + 8 * i + (lane >> 2);
        if (u < u1) {
            const int r = u / steps, step = u - r * steps, seg = MODE == GV_EXPERT_DOWN ? step / ksteps : 0;
            const int col = ((step - seg * ksteps) << 8) + (lane & 3) * 64;
            if (col < p.ldw) prefetch_l2(row_start(r, seg) - lane * 8 + col);
        }
    }
    constexpr int SG = 2;  // column groups per thread requested together
    float4 nw[SG];
    if (a.has_stage) {
        stream_coefs(a.st, coef);
#pragma unroll
        for (int i = 0; i < SG; ++i) {
            const int g = threadIdx.x + i * DG_THREADS;
            nw[i] = g < (a.st.ld >> 2) ? __ldg(reinterpret_cast<const float4*>(a.st.norm) + g) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    if (!late) {
        pdl_wait();
        pdl_trigger();
    }
    __syncthreads();

    if (a.has_stage) {
        const StreamStage& s = a.st;
        const int n4 = s.ld >> 2;
        int k = 0;
        for (int r = 0; r < R; ++r) {
            float ss = 0.f;
            for (int g0 = threadIdx.x; g0 < (kx >> 2); g0 += SG * DG_THREADS) {
                StreamGroup<S> sg[SG];
#pragma unroll
                for (int i = 0; i < SG; ++i)
                    if (g0 + i * DG_THREADS < n4) sg[i].template load<false>(s, r, g0 + i * DG_THREADS, nullptr, nullptr);
#pragma unroll
                for (int i = 0; i < SG; ++i) {
                    const int g = g0 + i * DG_THREADS;
                    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (g < n4) {
                        u = sg[i].finish(s, coef, r, g, g % gridDim.x == blockIdx.x);
                        ss += S == 1 && s.norm_b ? u.x + u.y + u.z + u.w : u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
                    }
                    if (g < (kx >> 2)) {
                        *reinterpret_cast<float4*>(xs + r * kx + dg_slot(g << 2)) = u;
                        if (MODE == GV_DUAL && g >= n4) *reinterpret_cast<float4*>(xs + (R + r) * kx + dg_slot(g << 2)) = u;
                    }
                }
            }
            ss = block_sum_alt(ss, red, k);
            float mean = 0.f;
            if (S == 1 && s.norm_b) {
                mean = ss / (float)s.n;
                ss = 0.f;
                for (int g = threadIdx.x; g < n4; g += DG_THREADS)
                    ss += squared_deviations(*reinterpret_cast<const float4*>(xs + r * kx + dg_slot(g << 2)), mean, g, s.n);
                ss = block_sum_alt(ss, red, k);
            }
            const float inv = 1.0f / sqrtf(ss / (float)s.n + s.eps);
            auto scale = [&](int g, const float4 w) {  // own groups
                float4* q = reinterpret_cast<float4*>(xs + r * kx + dg_slot(g << 2));
                const float4 u = *q;
                float4 v = norm_group(u, mean, inv, w, S == 1 ? s.norm_b : nullptr, g);
                if (!p.f32) v = make_float4(round_bf16(v.x), round_bf16(v.y), round_bf16(v.z), round_bf16(v.w));
                *q = v;
                if constexpr (MODE == GV_DUAL) {
                    v = norm_group(u, mean, inv, s.norm2, s.norm2_b, g);
                    if (g % gridDim.x == blockIdx.x) {
                        if (s.h_f32)
                            reinterpret_cast<float4*>(static_cast<float*>(s.h2) + (size_t)r * s.ldh)[g] = v;
                        else
                            reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(s.h2) + (size_t)r * s.ldh)[g] = float4_to_bf16x4(v);
                    }
                    if (!p.f32) v = make_float4(round_bf16(v.x), round_bf16(v.y), round_bf16(v.z), round_bf16(v.w));
                    *reinterpret_cast<float4*>(xs + (R + r) * kx + dg_slot(g << 2)) = v;
                }
            };
#pragma unroll
            for (int i = 0; i < SG; ++i)
                if ((int)threadIdx.x + i * DG_THREADS < n4) scale(threadIdx.x + i * DG_THREADS, nw[i]);
            for (int g = threadIdx.x + SG * DG_THREADS; g < n4; g += DG_THREADS)
                scale(g, __ldg(reinterpret_cast<const float4*>(s.norm) + g));
        }
    } else {
        constexpr int XG = 4;  // column groups per thread requested together
        constexpr bool RAW = MODE == GV_GROUPS || MODE == GV_NORMED;
        const bool wide = p.f32 || (RAW && p.x_raw);  // float32 rows
        const int n4 = kx >> 2;
        // first element of staged row q (of x's rows; of a token's choices)
        auto row_of = [&](int q) {
            if constexpr (MODE == GV_GROUPS) return (size_t)q * p.ldx + (size_t)y * p.gx_col;
            if constexpr (MODE == GV_EXPERT_UP) return (size_t)(y / a.route.top) * p.ldx;
            if constexpr (MODE == GV_EXPERT_DOWN) return ((size_t)y * a.route.top + q) * p.ldx;
            return (size_t)q * p.ldx;
        };
        auto request = [&](int q, int g) {
            if ((g << 2) >= p.k) return make_float4(0.f, 0.f, 0.f, 0.f);
            if (wide) return __ldcg(reinterpret_cast<const float4*>(static_cast<const float*>(p.x) + row_of(q)) + g);
            return bf16x4_to_float4(__ldcg(reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p.x) + row_of(q)) + g));
        };
        auto put = [&](int q, int g, float4 v) {
            const int c = g << 2;
            if (c + 1 >= p.k) v.y = 0.f;  // (pad columns of the row may hold another product's values)
            if (c + 2 >= p.k) v.z = 0.f;
            if (c + 3 >= p.k) v.w = 0.f;
            if constexpr (MODE == GV_EXPERT_DOWN) {
                const float gain = s_weight[q];
                v = make_float4(v.x * gain, v.y * gain, v.z * gain, v.w * gain);
            }
            if (MODE == GV_GROUPS && p.x_raw && !p.f32) v = make_float4(round_bf16(v.x), round_bf16(v.y), round_bf16(v.z), round_bf16(v.w));
            *reinterpret_cast<float4*>(xs + q * kx + dg_slot(c)) = v;
        };
        if constexpr (MODE == GV_EXPERT_DOWN) {  // short rows: requests run on from one to the next
            for (int i0 = threadIdx.x; i0 < segs * n4; i0 += XG * DG_THREADS) {
                float4 f[XG];
#pragma unroll
                for (int i = 0; i < XG; ++i)
                    if (i0 + i * DG_THREADS < segs * n4) f[i] = request((i0 + i * DG_THREADS) / n4, (i0 + i * DG_THREADS) % n4);
#pragma unroll
                for (int i = 0; i < XG; ++i)
                    if (i0 + i * DG_THREADS < segs * n4) put((i0 + i * DG_THREADS) / n4, (i0 + i * DG_THREADS) % n4, f[i]);
            }
        } else {
            for (int r = 0; r < R; ++r)
                for (int g0 = threadIdx.x; g0 < n4; g0 += XG * DG_THREADS) {
                    float4 f[XG];
#pragma unroll
                    for (int i = 0; i < XG; ++i) f[i] = request(r, g0 + i * DG_THREADS);
#pragma unroll
                    for (int i = 0; i < XG; ++i)
                        if (g0 + i * DG_THREADS < n4) put(r, g0 + i * DG_THREADS, f[i]);
                }
        }
        if constexpr (MODE == GV_NORMED) {
            int k = 0;
            for (int r = 0; r < R; ++r) {
                float ss = 0.f;
                for (int g = threadIdx.x; g < n4; g += DG_THREADS) {  // own groups
                    const float4 u = *reinterpret_cast<const float4*>(xs + r * kx + dg_slot(g << 2));
                    ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
                }
                ss = block_sum_alt(ss, red, k);
                const float inv = 1.0f / sqrtf(ss / (float)p.k + p.x_eps);
                for (int g = threadIdx.x; (g << 2) < p.k; g += DG_THREADS) {
                    float4* v = reinterpret_cast<float4*>(xs + r * kx + dg_slot(g << 2));
                    float4 u = norm_group(*v, 0.f, inv, p.x_norm, nullptr, g);
                    if (!p.f32) u = make_float4(round_bf16(u.x), round_bf16(u.y), round_bf16(u.z), round_bf16(u.w));
                    *v = u;
                }
            }
        }
    }
    __syncthreads();

    float acc[R], acc2[R];
#pragma unroll
    for (int r = 0; r < R; ++r) acc[r] = acc2[r] = 0.f;
    int crow = u0 / steps, cstep = u0 - crow * steps, cu = u0;
    auto flush = [&]() {
        const int slot = warp - (crow * steps) / upw;
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const float t = warp_sum(acc[r] + acc2[r]);
            if (lane == 0) part[((size_t)crow * a.slots + slot) * R + r] = t;
            acc[r] = acc2[r] = 0.f;
        }
    };
    // rows of x that output row `row` (of this CTA) multiplies
    auto operand = [&](int row) -> const float* {
        if constexpr (MODE == GV_DUAL) return xs + (n0 + row >= p.n ? R * kx : 0);
        return xs;
    };
    auto mac = [&](const uint4& w, const float* x) {
        const float4 wlo = bf16x4_to_float4(make_uint2(w.x, w.y)), whi = bf16x4_to_float4(make_uint2(w.z, w.w));
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const float4 xa = *reinterpret_cast<const float4*>(x + r * kx), xb = *reinterpret_cast<const float4*>(x + r * kx + 128);
            acc[r] += wlo.x * xa.x;
            acc2[r] += whi.x * xb.x;
            acc[r] += wlo.y * xa.y;
            acc2[r] += whi.y * xb.y;
            acc[r] += wlo.z * xa.z;
            acc2[r] += whi.z * xb.z;
            acc[r] += wlo.w * xa.w;
            acc2[r] += whi.w * xb.w;
        }
    };
    auto consume = [&](const uint4 (&w)[DG_U]) {
        const float* x = operand(crow) + (cstep << 8) + lane * 4;
        if (cu + DG_U <= u1 && cstep + DG_U <= steps) {  // one row, the whole batch (warp-uniform)
#pragma unroll
            for (int j = 0; j < DG_U; ++j) mac(w[j], x + (j << 8));
            cu += DG_U;
            cstep += DG_U;
            if (cstep == steps) {
                flush();
                cstep = 0;
                ++crow;
            } else if (cu == u1) {
                flush();
            }
            return;
        }
#pragma unroll
        for (int j = 0; j < DG_U; ++j) {
            if (cu < u1) {
                mac(w[j], operand(crow) + (cstep << 8) + lane * 4);
                ++cu;
                if (++cstep == steps) {
                    flush();
                    cstep = 0;
                    ++crow;
                } else if (cu == u1) {
                    flush();
                }
            }
        }
    };
    fetch(wb);
    while (cu < u1) {
        consume(wa);
        fetch(wa);
        consume(wb);
        fetch(wb);
    }
    __syncthreads();

    // ---- a row's shares in warp order, then the output
    auto total = [&](int row, int r) {
        const int first = (row * steps) / upw, last = ((row + 1) * steps - 1) / upw;
        float t = 0.f;
        for (int w = first; w <= last; ++w) t += part[((size_t)row * a.slots + w - first) * R + r];
        return t;
    };
    for (int i = threadIdx.x; i < (n1 - n0) * R; i += DG_THREADS) {
        const int r = i / (n1 - n0), o = i - r * (n1 - n0);
        auto put = [&](size_t at, float v) {
            if (p.f32)
                static_cast<float*>(p.a)[at] = v;
            else
                static_cast<__nv_bfloat16*>(p.a)[at] = __float2bfloat16_rn(v);
        };
        if (gated) {
            const float v = gate_act(p.act, total(2 * o, r)) * total(2 * o + 1, r);
            put((size_t)(MODE == GV_EXPERT_UP ? y : r) * p.lda + n0 + o, v);
        } else if (MODE == GV_GROUPS) {
            float v = total(o, r);
            if (p.head_gate) v *= sigmoid(__ldcg(p.head_gate + (size_t)r * p.ld_head_gate + y));
            put((size_t)r * p.lda + (size_t)y * p.gy_col + n0 + o, v);
        } else if (MODE == GV_DUAL && n0 + o >= p.n) {
            p.y2[(size_t)r * p.ldy2 + n0 + o - p.n] = total(o, r);
        } else {
            p.y[(size_t)(MODE == GV_EXPERT_DOWN ? y : r) * p.ldy + n0 + o] = total(o, r);
        }
    }
}

static int dg_mode(const DenseProduct& p) {
    if (p.route) return p.epilogue == DENSE_GATED ? GV_EXPERT_UP : GV_EXPERT_DOWN;
    if (p.groups) return GV_GROUPS;
    if (p.x_norm) return GV_NORMED;
    return p.stage && p.stage->norm2 ? GV_DUAL : GV_PLAIN;
}

static size_t dg_plan(const DenseProduct& p, int rows, int* grid, int* slots) {
    const int mode = dg_mode(p), kx = (p.k + 255) & ~255, pair = p.epilogue == DENSE_GATED ? 2 : 1;
    const int top = p.route ? p.route->top : 1, steps = kx / 256 * (mode == GV_EXPERT_DOWN ? top : 1);
    const int n = mode == GV_DUAL ? p.n + p.n2 : p.n, planes = mode == GV_GROUPS ? p.groups : mode == GV_EXPERT_UP ? rows * top : mode == GV_EXPERT_DOWN ? rows : 1;
    const int ctas = DG_CTAS / planes < 1 ? 1 : DG_CTAS / planes, r = p.route ? 1 : rows;
    *grid = n < ctas ? n : ctas;
    const int lo = n / *grid * pair, hi = (n + *grid - 1) / *grid * pair;
    const int upw = (lo * steps + DG_WARPS - 1) / DG_WARPS;
    *slots = (steps + upw - 1) / upw + 1;
    const int xrows = mode == GV_DUAL ? 2 * r : mode == GV_EXPERT_DOWN ? top : r;
    return ((size_t)xrows * kx + (size_t)hi * *slots * r) * sizeof(float);
}

bool dense_gemv_supported(const DenseProduct& p, int rows) {
    int g, s;
    if (p.groups > 65535 || p.epilogue == DENSE_QKV || p.epilogue == DENSE_ROPE || (p.route && (p.route->top > EXPERT_TOP_MAX || p.route->top < 1))) return false;
    // (what a stage adds up and norms beyond one stream's share is the stage kernel's)
    if (p.stage && (p.stage->slots || (p.stage->streams != 1 && (p.stage->norm_b || p.stage->y2)))) return false;
    return rows >= 1 && rows <= DENSE_FEW_ROWS && p.n > 0 && p.k > 0 && dg_plan(p, rows, &g, &s) <= DG_SMEM_MAX;
}

template <int R, int S, int MODE>
static int dg_configure() {
    RB_CUDA(cudaFuncSetAttribute(dense_gemv_kernel<R, S, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DG_SMEM_MAX));
    return ROTOR_B200_OK;
}
template <int R>
static int dg_configure_all() {
    int rc;
    if ((rc = dg_configure<R, 0, GV_PLAIN>()) || (rc = dg_configure<R, 1, GV_PLAIN>()) || (rc = dg_configure<R, 2, GV_PLAIN>()) ||
        (rc = dg_configure<R, 3, GV_PLAIN>()) || (rc = dg_configure<R, 4, GV_PLAIN>()) || (rc = dg_configure<R, 1, GV_DUAL>()) ||
        (rc = dg_configure<R, 1, GV_GROUPS>()) || (rc = dg_configure<R, 1, GV_NORMED>()))
        return rc;
    return ROTOR_B200_OK;
}
int configure_dense_gemv() {
    int rc;
    if ((rc = dg_configure_all<1>()) || (rc = dg_configure_all<2>()) || (rc = dg_configure_all<3>()) || (rc = dg_configure_all<4>()) ||
        (rc = dg_configure<1, 1, GV_EXPERT_UP>()) || (rc = dg_configure<1, 1, GV_EXPERT_DOWN>()))
        return rc;
    return ROTOR_B200_OK;
}

template <int R>
static int dg_launch(const DenseGemvArgs& a, int mode, int grid, size_t smem, cudaStream_t st) {
    const dim3 g(grid, mode == GV_GROUPS ? a.p.groups : 1), b(DG_THREADS);
    if (mode == GV_GROUPS) return launch_chained(dense_gemv_kernel<R, 1, GV_GROUPS>, g, b, smem, st, 1, a);
    if (mode == GV_NORMED) return launch_chained(dense_gemv_kernel<R, 1, GV_NORMED>, g, b, smem, st, 1, a);
    if (mode == GV_DUAL) return launch_chained(dense_gemv_kernel<R, 1, GV_DUAL>, g, b, smem, st, 1, a);
    switch (a.has_stage ? a.st.streams : 1) {
        case 1: return launch_chained(dense_gemv_kernel<R, 1, GV_PLAIN>, g, b, smem, st, 1, a);
        case 2: return launch_chained(dense_gemv_kernel<R, 2, GV_PLAIN>, g, b, smem, st, 1, a);
        case 3: return launch_chained(dense_gemv_kernel<R, 3, GV_PLAIN>, g, b, smem, st, 1, a);
        case 4: return launch_chained(dense_gemv_kernel<R, 4, GV_PLAIN>, g, b, smem, st, 1, a);
        default: return launch_chained(dense_gemv_kernel<R, 0, GV_PLAIN>, g, b, smem, st, 1, a);
    }
}

int launch_dense_gemv(const DenseProduct& p, int rows, cudaStream_t st) {
    if (!dense_gemv_supported(p, rows)) return ROTOR_B200_ERR_SHAPE;
    const int mode = dg_mode(p);
    RB_REQUIRE(p.w && p.ldw % 8 == 0 && p.ldw >= p.k && (p.stage || (p.x && p.ldx % 4 == 0)));
    RB_REQUIRE(p.epilogue == DENSE_GATED || mode == GV_GROUPS ? p.a != nullptr : p.y != nullptr);
    RB_REQUIRE(mode != GV_GROUPS || (p.epilogue == DENSE_HALF && p.gx_col % 4 == 0 && !p.stage));
    RB_REQUIRE(!p.route || (p.route->logits && p.route->top <= p.route->experts && !p.stage && !p.x_norm));
    RB_REQUIRE(!p.x_norm || (p.x_raw && !p.stage && mode == GV_NORMED));
    RB_REQUIRE(!p.x_raw || mode == GV_NORMED || mode == GV_GROUPS);
    DenseGemvArgs a = {};
    a.p = p;
    if (p.route) a.route = *p.route;
    a.rows = rows;
    a.has_stage = p.stage != nullptr;
    if (p.stage) {
        RB_REQUIRE(p.stage->streams >= 1 && p.stage->streams <= STREAMS_MAX && p.stage->n == p.k && p.stage->x_out &&
                   !p.stage->row_map);
        RB_REQUIRE(mode != GV_DUAL || (p.stage->streams == 1 && p.stage->h2 && (p.n2 == 0 || (p.w2 && p.y2))));
        RB_REQUIRE(!p.stage->norm2 || (p.stage->norm_b != nullptr) == (p.stage->norm2_b != nullptr));
        a.st = *p.stage;
    }
    int grid, slots;
    const size_t smem = dg_plan(p, rows, &grid, &slots);
    a.slots = slots;
    if (mode == GV_EXPERT_UP)
        return launch_chained(dense_gemv_kernel<1, 1, GV_EXPERT_UP>, dim3(grid, rows * p.route->top), dim3(DG_THREADS), smem, st, 1, a);
    if (mode == GV_EXPERT_DOWN)
        return launch_chained(dense_gemv_kernel<1, 1, GV_EXPERT_DOWN>, dim3(grid, rows), dim3(DG_THREADS), smem, st, 1, a);
    switch (rows) {
        case 1: return dg_launch<1>(a, mode, grid, smem, st);
        case 2: return dg_launch<2>(a, mode, grid, smem, st);
        case 3: return dg_launch<3>(a, mode, grid, smem, st);
        default: return dg_launch<4>(a, mode, grid, smem, st);
    }
}

}  // namespace rb

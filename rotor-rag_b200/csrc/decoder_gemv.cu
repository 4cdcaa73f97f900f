// Dense products of up to four rows (generation steps): y = x W^T with bf16 weights, bound by the weight
// stream, with the residual stage that produces x fused into the prologue and the gating into the end.
//
// Grid: two CTAs per SM, each owning a contiguous run of output rows (a gated product: of gate / up pairs).
// The run's work is a list of units (output row, 256 columns); the CTA's warps take equal contiguous
// shares of that list, so that rows are split across warps where that is what balances them, and the
// shares of a row are added in warp order (fixed order: repeated runs give identical bits).  A unit is
// one 128-bit weight load per lane; loads run a batch ahead of the arithmetic, and the first batches
// are requested before the programmatic-launch wait.
#include "decoder.cuh"

namespace rb {

constexpr int DG_THREADS = 512, DG_WARPS = DG_THREADS / 32, DG_CTAS = 296;
constexpr int DG_U = 4;                       // units per load batch
constexpr int DG_AHEAD = 16;                  // units requested into L2 ahead of the launch wait
constexpr size_t DG_SMEM_MAX = 200 * 1024;

struct DenseGemvArgs {
    DenseProduct p;
    StreamStage st;
    int has_stage, rows, slots, max_rows;
};

// Column i (a multiple of 4) of a staged row: the two halves of a lane's eight columns sit 128 floats
// apart, which makes both 128-bit reads of a unit free of bank conflicts.
__device__ __forceinline__ int dg_slot(int i) { return (i & ~255) + ((i >> 2) & 1) * 128 + ((i & 255) >> 3) * 4; }

template <int R, int S>
__global__ void __launch_bounds__(DG_THREADS, R <= 2 ? 2 : 1) dense_gemv_kernel(const __grid_constant__ DenseGemvArgs a) {
    const DenseProduct& p = a.p;
    extern __shared__ __align__(16) float sm[];
    __shared__ float coef[STREAMS_MAX * STREAMS_MAX + 2 * STREAMS_MAX], red[64];
    const int kx = (p.k + 255) & ~255, steps = kx >> 8;
    float* xs = sm;                 // [R][kx]
    float* part = sm + R * kx;      // [local row][slot][R]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const bool gated = p.epilogue == DENSE_GATED;
    const int n0 = (int)((long long)blockIdx.x * p.n / gridDim.x), n1 = (int)((long long)(blockIdx.x + 1) * p.n / gridDim.x);
    const int lr = (n1 - n0) * (gated ? 2 : 1);
    const int units = lr * steps, upw = max(1, (units + DG_WARPS - 1) / DG_WARPS);
    const int u0 = min(units, warp * upw), u1 = min(units, u0 + upw);

    // load cursor, a batch ahead of the arithmetic cursor
    auto row_start = [&](int r) {
        const int row = gated ? (r & 1) * p.n + n0 + (r >> 1) : n0 + r;
        return p.w + (size_t)row * p.ldw + lane * 8;
    };
    int lrow = u0 / steps, lstep = u0 - lrow * steps, lu = u0, lcol = (lstep << 8) + lane * 8;
    const __nv_bfloat16* lp = row_start(lrow) + (lstep << 8);
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
                lcol = lane * 8;
                lp = row_start(++lrow);
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
            const int r = u / steps, col = ((u - r * steps) << 8) + (lane & 3) * 64;
            if (col < p.ldw) prefetch_l2(row_start(r) - lane * 8 + col);
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
    pdl_wait();
    pdl_trigger();
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
                    if (g0 + i * DG_THREADS < n4) sg[i].load(s, r, g0 + i * DG_THREADS);
#pragma unroll
                for (int i = 0; i < SG; ++i) {
                    const int g = g0 + i * DG_THREADS;
                    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
                    if (g < n4) {
                        u = sg[i].finish(s, coef, r, g, g % gridDim.x == blockIdx.x);
                        ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
                    }
                    if (g < (kx >> 2)) *reinterpret_cast<float4*>(xs + r * kx + dg_slot(g << 2)) = u;
                }
            }
            ss = block_sum_alt(ss, red, k);
            const float inv = 1.0f / sqrtf(ss / (float)s.n + s.eps);
            auto scale = [&](int g, const float4 w) {  // own groups
                float4* q = reinterpret_cast<float4*>(xs + r * kx + dg_slot(g << 2));
                float4 v = *q;
                v = make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w);
                if (!p.f32) v = make_float4(round_bf16(v.x), round_bf16(v.y), round_bf16(v.z), round_bf16(v.w));
                *q = v;
            };
#pragma unroll
            for (int i = 0; i < SG; ++i)
                if ((int)threadIdx.x + i * DG_THREADS < n4) scale(threadIdx.x + i * DG_THREADS, nw[i]);
            for (int g = threadIdx.x + SG * DG_THREADS; g < n4; g += DG_THREADS)
                scale(g, __ldg(reinterpret_cast<const float4*>(s.norm) + g));
        }
    } else {
        constexpr int XG = 4;
        for (int r = 0; r < R; ++r)
            for (int g0 = threadIdx.x; g0 < (kx >> 2); g0 += XG * DG_THREADS) {
                float4 f[XG];
#pragma unroll
                for (int i = 0; i < XG; ++i) {
                    const int g = g0 + i * DG_THREADS;
                    f[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                    if ((g << 2) >= p.k) continue;
                    if (p.f32)
                        f[i] = __ldcg(reinterpret_cast<const float4*>(static_cast<const float*>(p.x) + (size_t)r * p.ldx) + g);
                    else
                        f[i] = bf16x4_to_float4(__ldcg(reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p.x) + (size_t)r * p.ldx) + g));
                }
#pragma unroll
                for (int i = 0; i < XG; ++i) {
                    const int c = (g0 + i * DG_THREADS) << 2;
                    if (c >= kx) continue;
                    if (c + 1 >= p.k) f[i].y = 0.f;  // (pad columns of the row may hold another product's values)
                    if (c + 2 >= p.k) f[i].z = 0.f;
                    if (c + 3 >= p.k) f[i].w = 0.f;
                    *reinterpret_cast<float4*>(xs + r * kx + dg_slot(c)) = f[i];
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
        const float* x = xs + (cstep << 8) + lane * 4;
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
                mac(w[j], xs + (cstep << 8) + lane * 4);
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
        if (gated) {
            const float v = gelu_tanh(total(2 * o, r)) * total(2 * o + 1, r);
            if (p.f32)
                static_cast<float*>(p.a)[(size_t)r * p.lda + n0 + o] = v;
            else
                static_cast<__nv_bfloat16*>(p.a)[(size_t)r * p.lda + n0 + o] = __float2bfloat16_rn(v);
        } else {
            p.y[(size_t)r * p.ldy + n0 + o] = total(o, r);
        }
    }
}

static size_t dg_plan(const DenseProduct& p, int rows, int* grid, int* slots) {
    const int kx = (p.k + 255) & ~255, steps = kx / 256, pair = p.epilogue == DENSE_GATED ? 2 : 1;
    *grid = p.n < DG_CTAS ? p.n : DG_CTAS;
    const int lo = p.n / *grid * pair, hi = (p.n + *grid - 1) / *grid * pair;
    const int upw = (lo * steps + DG_WARPS - 1) / DG_WARPS;
    *slots = (steps + upw - 1) / upw + 1;
    return ((size_t)rows * kx + (size_t)hi * *slots * rows) * sizeof(float);
}

bool dense_gemv_supported(const DenseProduct& p, int rows) {
    int g, s;
    return rows >= 1 && rows <= DENSE_FEW_ROWS && p.n > 0 && p.k > 0 && dg_plan(p, rows, &g, &s) <= DG_SMEM_MAX;
}

template <int R, int S>
static int dg_configure() {
    RB_CUDA(cudaFuncSetAttribute(dense_gemv_kernel<R, S>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DG_SMEM_MAX));
    return ROTOR_B200_OK;
}
template <int R>
static int dg_configure_all() {
    int rc;
    if ((rc = dg_configure<R, 0>()) || (rc = dg_configure<R, 1>()) || (rc = dg_configure<R, 2>()) || (rc = dg_configure<R, 3>()) ||
        (rc = dg_configure<R, 4>()))
        return rc;
    return ROTOR_B200_OK;
}
int configure_dense_gemv() {
    int rc;
    if ((rc = dg_configure_all<1>()) || (rc = dg_configure_all<2>()) || (rc = dg_configure_all<3>()) || (rc = dg_configure_all<4>()))
        return rc;
    return ROTOR_B200_OK;
}

template <int R>
static int dg_launch(const DenseGemvArgs& a, int grid, size_t smem, cudaStream_t st) {
    const dim3 g(grid), b(DG_THREADS);
    switch (a.has_stage ? a.st.streams : 1) {
        case 1: return launch_chained(dense_gemv_kernel<R, 1>, g, b, smem, st, 1, a);
        case 2: return launch_chained(dense_gemv_kernel<R, 2>, g, b, smem, st, 1, a);
        case 3: return launch_chained(dense_gemv_kernel<R, 3>, g, b, smem, st, 1, a);
        case 4: return launch_chained(dense_gemv_kernel<R, 4>, g, b, smem, st, 1, a);
        default: return launch_chained(dense_gemv_kernel<R, 0>, g, b, smem, st, 1, a);
    }
}

int launch_dense_gemv(const DenseProduct& p, int rows, cudaStream_t st) {
    if (!dense_gemv_supported(p, rows)) return ROTOR_B200_ERR_SHAPE;
    RB_REQUIRE(p.w && p.ldw % 8 == 0 && p.ldw >= p.k && (p.stage || (p.x && p.ldx % 4 == 0)));
    RB_REQUIRE(p.epilogue == DENSE_GATED ? p.a != nullptr : p.y != nullptr);
    DenseGemvArgs a = {};
    a.p = p;
    a.rows = rows;
    a.has_stage = p.stage != nullptr;
    if (p.stage) {
        RB_REQUIRE(p.stage->streams >= 1 && p.stage->streams <= STREAMS_MAX && p.stage->n == p.k && p.stage->x_out &&
                   !p.stage->row_map);
        a.st = *p.stage;
    }
    int grid, slots;
    const size_t smem = dg_plan(p, rows, &grid, &slots);
    a.slots = slots;
    switch (rows) {
        case 1: return dg_launch<1>(a, grid, smem, st);
        case 2: return dg_launch<2>(a, grid, smem, st);
        case 3: return dg_launch<3>(a, grid, smem, st);
        default: return dg_launch<4>(a, grid, smem, st);
    }
}

}  // namespace rb

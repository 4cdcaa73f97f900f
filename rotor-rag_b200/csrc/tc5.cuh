// Fifth-generation tensor-core pieces shared by the kernels that use tcgen05: bounded mbarrier
// waits, operand descriptors, MMA issue and commit, tensor-memory loads and stores, TMA loads and
// the read-back that turns tensor-memory lanes into whole output rows.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>

#include "gemv_core.cuh"

namespace rb {

constexpr long long T5_SPIN_CYCLES = 400000000LL;  // about 0.2 s

__device__ __forceinline__ bool t5_wait(uint32_t bar, uint32_t parity, volatile int* abort_flag, unsigned* status,
                                        unsigned code) {
    long long t0 = 0;
    for (int it = 0;; ++it) {
        uint32_t ok;
        asm volatile(
            "{ .reg .pred p; mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2; selp.u32 %0, 1, 0, p; }"
            : "=r"(ok)
            : "r"(bar), "r"(parity)
            : "memory");
        if (ok) return true;
        if (*abort_flag) return false;
        if (it == 0) t0 = clock64();
        if (clock64() - t0 > T5_SPIN_CYCLES) {
            *abort_flag = 1;
            atomicExch(status, code);
            return false;
        }
    }
}

// Shared-memory matrix descriptor, K-major, 128-byte swizzle: 8-row groups 1024 bytes apart.
__device__ __forceinline__ uint64_t t5_desc(uint32_t smem_addr) {
    return (uint64_t)((smem_addr >> 4) & 0x3fffu) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) |
           (2ull << 61);
}

__device__ __forceinline__ void t5_ld32(uint32_t taddr, uint32_t (&v)[32]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
        "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
        "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
        : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]),
          "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]), "=r"(v[16]),
          "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]), "=r"(v[24]),
          "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
        : "r"(taddr));
}

// Read-back store of a warp's 32 tokens x 32 values (lane = token after tcgen05.ld) as whole 128-byte
// rows: through a per-warp shared-memory block (32 rows of 144 bytes: conflict-free both ways) so that
// one store instruction covers four tokens' rows (four lines) instead of one 16-byte piece of 32
// different lines.  dst0: address of token tok_base's first value; tokens at and beyond ntok are skipped.
constexpr uint32_t T5_XPOSE_BYTES = 32 * 144;
__device__ __forceinline__ void t5_store_rows(uint32_t stage, const uint32_t (&v)[32], void* dst0, size_t row_bytes,
                                              int tok_base, int ntok, int lane) {
#pragma unroll
    for (int q = 0; q < 8; ++q)
        asm volatile("st.shared.v4.u32 [%0], {%1, %2, %3, %4};" ::"r"(stage + (uint32_t)lane * 144u + 16u * q),
                     "r"(v[4 * q]), "r"(v[4 * q + 1]), "r"(v[4 * q + 2]), "r"(v[4 * q + 3])
                     : "memory");
    __syncwarp();
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int tl = 4 * i + (lane >> 3);
        uint4 w;
        asm volatile("ld.shared.v4.u32 {%0, %1, %2, %3}, [%4];"
                     : "=r"(w.x), "=r"(w.y), "=r"(w.z), "=r"(w.w)
                     : "r"(stage + (uint32_t)tl * 144u + 16u * (lane & 7)));
        if (tok_base + tl < ntok)
            *reinterpret_cast<uint4*>(static_cast<unsigned char*>(dst0) + (size_t)tl * row_bytes + 16 * (lane & 7)) = w;
    }
    __syncwarp();  // the block is rewritten by the warp's next item
}

// The same with a destination per token: dst_of(tl) is the address of token tok_base + tl's 128 bytes
// (null = skip).
template <typename F>
__device__ __forceinline__ void t5_store_rows_to(uint32_t stage, const uint32_t (&v)[32], int lane, F dst_of) {
#pragma unroll
    for (int q = 0; q < 8; ++q)
        asm volatile("st.shared.v4.u32 [%0], {%1, %2, %3, %4};" ::"r"(stage + (uint32_t)lane * 144u + 16u * q),
                     "r"(v[4 * q]), "r"(v[4 * q + 1]), "r"(v[4 * q + 2]), "r"(v[4 * q + 3])
                     : "memory");
    __syncwarp();
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int tl = 4 * i + (lane >> 3);
        uint4 w;
        asm volatile("ld.shared.v4.u32 {%0, %1, %2, %3}, [%4];"
                     : "=r"(w.x), "=r"(w.y), "=r"(w.z), "=r"(w.w)
                     : "r"(stage + (uint32_t)tl * 144u + 16u * (lane & 7)));
        unsigned char* d = static_cast<unsigned char*>(dst_of(tl));
        if (d) *reinterpret_cast<uint4*>(d + 16 * (lane & 7)) = w;
    }
    __syncwarp();
}

// The 32 tokens x 64 bytes counterpart of t5_store_rows_to: dst_of(tl) is the address of token tl's 64 bytes.
template <typename F>
__device__ __forceinline__ void t5_store_half_rows_to(uint32_t stage, const uint32_t (&v)[16], int lane, F dst_of) {
#pragma unroll
    for (int q = 0; q < 4; ++q)
        asm volatile("st.shared.v4.u32 [%0], {%1, %2, %3, %4};" ::"r"(stage + (uint32_t)lane * 80u + 16u * q),
                     "r"(v[4 * q]), "r"(v[4 * q + 1]), "r"(v[4 * q + 2]), "r"(v[4 * q + 3])
                     : "memory");
    __syncwarp();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int tl = 8 * i + (lane >> 2);
        uint4 w;
        asm volatile("ld.shared.v4.u32 {%0, %1, %2, %3}, [%4];"
                     : "=r"(w.x), "=r"(w.y), "=r"(w.z), "=r"(w.w)
                     : "r"(stage + (uint32_t)tl * 80u + 16u * (lane & 3)));
        unsigned char* d = static_cast<unsigned char*>(dst_of(tl));
        if (d) *reinterpret_cast<uint4*>(d + 16 * (lane & 3)) = w;
    }
    __syncwarp();
}
__device__ __forceinline__ uint32_t t5_pack(float a, float b) {  // bf16x2, first value in the low half
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ void t5_st32(uint32_t taddr, const uint32_t (&v)[32]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
        "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};" ::"r"(taddr),
        "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]),
        "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]), "r"(v[16]), "r"(v[17]), "r"(v[18]),
        "r"(v[19]), "r"(v[20]), "r"(v[21]), "r"(v[22]), "r"(v[23]), "r"(v[24]), "r"(v[25]), "r"(v[26]), "r"(v[27]),
        "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31])
        : "memory");
}

// Descriptor of an operand stored with its M or N dimension contiguous, 128-byte swizzle: panels of 64
// elements `panel_bytes` apart, eight K rows of a panel in 1024 bytes.
__device__ __forceinline__ uint64_t t5_desc_mn(uint32_t smem_addr, uint32_t panel_bytes) {
    return (uint64_t)((smem_addr >> 4) & 0x3fffu) | ((uint64_t)(panel_bytes >> 4) << 16) |
           ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}

// Instruction descriptor of kind::f16 with bf16 operands and float32 accumulation; b_mn: the B operand is
// stored with N contiguous.
__host__ __device__ constexpr uint32_t t5_idesc_bf16(int m, int n, bool b_mn = false) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((b_mn ? 1u : 0u) << 16) | ((uint32_t)(n >> 3) << 17) |
           ((uint32_t)(m >> 4) << 24);
}

__device__ __forceinline__ void t5_mma_ss(uint32_t d_tmem, uint64_t da, uint64_t db, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t"
        ".reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, {%5, %5, %5, %5}, p;\n\t"
        "}\n" ::"r"(d_tmem),
        "l"(da), "l"(db), "r"(idesc), "r"(accumulate), "r"(0u)
        : "memory");
}
// A operand in tensor memory
__device__ __forceinline__ void t5_mma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t db, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t"
        ".reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, {%5, %5, %5, %5}, p;\n\t"
        "}\n" ::"r"(d_tmem),
        "r"(a_tmem), "l"(db), "r"(idesc), "r"(accumulate), "r"(0u)
        : "memory");
}
__device__ __forceinline__ void t5_commit(uint32_t bar) {
    asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void t5_bar_init(uint32_t bar, uint32_t count) {
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count));
}
__device__ __forceinline__ void t5_bar_arrive(uint32_t bar) {
    asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void t5_bar_expect(uint32_t bar, uint32_t bytes) {
    asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
// Tiled load of this GPU's memory; x in elements, a multiple of 16 bytes.
__device__ __forceinline__ void t5_tma_2d(uint32_t dst, const CUtensorMap* map, int x, int y, uint32_t bar) {
    asm volatile(
        "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst),
        "l"(map), "r"(x), "r"(y), "r"(bar)
        : "memory");
}

typedef CUresult (*T5EncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                               const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                               CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
inline T5EncodeFn t5_encoder() {
    static T5EncodeFn fn = nullptr;
    if (!fn) {
        cudaDriverEntryPointQueryResult q;
        void* p = nullptr;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || !p ||
            q != cudaDriverEntryPointSuccess)
            return nullptr;
        fn = (T5EncodeFn)p;
    }
    return fn;
}
// bf16 matrix [rows][cols], row stride ld elements (a multiple of 8), box of 64 columns x box_rows rows,
// 128-byte swizzle; reads outside the matrix give zeros.
inline bool t5_map_bf16(CUtensorMap* map, const void* base, size_t rows, size_t cols, size_t ld, int box_rows) {
    T5EncodeFn enc = t5_encoder();
    const cuuint64_t gdim[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t gstride[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {64u, (cuuint32_t)box_rows};
    const cuuint32_t estride[2] = {1u, 1u};
    return enc && ((uintptr_t)base & 15) == 0 && ld % 8 == 0 &&
           enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), gdim, gstride, box, estride,
               CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
               CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

}  // namespace rb

// Y[M, N] = X[M, K] . W[N, K]^T on the fifth-generation tensor cores:
// bfloat16 operands brought into shared memory by TMA, tcgen05.mma issued by
// one thread with the accumulator in tensor memory, read back with tcgen05.ld
// for the epilogue.  This is the matrix product of prefill (M > 64); the
// decode step's product is gemm_small_m.cu.
//
// Both operands are K-major (X rows and W rows are contiguous in K), so a
// 128 x 64 tile of either is 128 rows of 128 bytes: exactly the 128-byte
// swizzle atom that TMA writes and the MMA's shared-memory descriptor reads.
//
// Block = one 128 x BN tile of Y, 6 warps:
//   warp 0   one lane issues the TMA loads of the K blocks into a ring of
//            STAGES buffers (full/empty mbarriers);
//   warp 1   allocates BN columns of tensor memory; one lane issues four
//            128 x BN x 16 MMAs per K block and commits to the stage's
//            "empty" barrier, at the end to the "accumulator ready" barrier;
//   warps 2-5 wait for the accumulator, read their 32 lanes (rows) of tensor
//            memory 32 columns at a time and write Y (store float32, store
//            bfloat16, or add into float32; optional bias).
// Two blocks fit one SM (3 stages of 32 KB each), so one block's epilogue
// overlaps the other's main loop.
//
// Every wait on an mbarrier is bounded: after about two seconds it gives up,
// raises the error flag that the host passes in, and the block still runs to
// its end and frees its tensor memory.  Rows past M or N and the tail of K are
// zero-filled by TMA and masked in the epilogue, so any M, N and any K that is
// a multiple of 8 (16-byte rows) work.
//
// Reference counterpart: quantized_matmul_rows, out[b, n] = sum_d in[b, d] W[n, d]
// (crates/mivi-quant/src/lib.rs:143-245).
#include "tc_common.cuh"

namespace {

constexpr int THREADS = 192;

#include "gemm_tc_store.cuh"

// The consuming end of a norm carried by products (see gemm_small_m.cu; null when unused): the rows of X
// still lack their norm's scale, so every row of the result is multiplied by
// rsqrt(sum of the row's partial sums / dim + eps).
struct RowScale {
    const float* part;                 // [rows][stride], n sums of squares per row
    int n, stride;
    float inv_dim, eps;
};
__device__ __forceinline__ float row_sum(const RowScale& rs, int row, int M) {
    float ss = 0.f;
    if (rs.part && row < M)
        for (int p = 0; p < rs.n; ++p) ss += rs.part[(size_t)row * rs.stride + p];
    return ss;
}
__device__ __forceinline__ void scale_chunk(unsigned (&r)[32], float sc) {
#pragma unroll
    for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * sc);
}

template <int BN, int STAGES>
struct SmemLayout {
    static constexpr int A_BYTES = BM * BK * 2, B_BYTES = BN * BK * 2;
    static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
    static constexpr int TILE_BYTES = STAGES * STAGE_BYTES;
    static constexpr int BAR_BYTES = (2 * STAGES + 1) * 8 + 8;
    static constexpr int TOTAL = TILE_BYTES + BAR_BYTES + 1024;      // 1024 for the manual alignment
};

template <int BN, int STAGES, int ACT>
__global__ void __launch_bounds__(THREADS)
gemm_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b,
               const float* __restrict__ bias, void* __restrict__ out, int mode, int M, int N, int K, int ldo,
               const RowScale rs, const RowWeights rw, int* __restrict__ err, const int* __restrict__ tile_group, int b_row_step,
               int b_k_step) {
    using L = SmemLayout<BN, STAGES>;
    // A grouped product (tile_group not null): the rows of X are sorted by group and padded so that no tile of 128
    // rows holds two groups; tile_group says which group a tile belongs to (negative: a spare tile, nothing to do),
    // and the group picks its part of W: b_row_step rows further down (W = the groups' matrices one below the
    // other) or b_k_step columns further along K (W = the groups' matrices side by side).  N and K are one group's.
    int group = 0;
    if (tile_group) {
        group = tile_group[blockIdx.y];
        if (group < 0) return;                     // the whole block, before any barrier or tensor memory exists
    }
    const int b_row0 = group * b_row_step, b_k0 = group * b_k_step;
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    unsigned long long* bars = (unsigned long long*)(smem + L::TILE_BYTES);
    unsigned* tmem_holder = (unsigned*)(bars + 2 * STAGES + 1);
    const unsigned full0 = smem_u32(bars), empty0 = full0 + 8 * STAGES, acc_bar = full0 + 16 * STAGES;
    const unsigned tiles0 = smem_u32(smem);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int m0 = blockIdx.y * BM, n0 = blockIdx.x * BN;
    const int kblocks = (K + BK - 1) / BK;

    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) {
            mbar_init(full0 + 8 * s, 1);
            mbar_init(empty0 + 8 * s, 1);
        }
        mbar_init(acc_bar, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                     ::"r"(smem_u32(tmem_holder)), "r"((unsigned)BN) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const unsigned tmem_base = *tmem_holder;

    if (warp == 0) {
        if (lane == 0) {
            for (int kb = 0; kb < kblocks; ++kb) {
                const int s = kb % STAGES;
                const unsigned phase = (unsigned)(kb / STAGES) & 1u;
                if (!mbar_wait(empty0 + 8 * s, phase ^ 1u, err, 1)) break;
                mbar_expect_tx(full0 + 8 * s, L::STAGE_BYTES);
                const unsigned a_dst = tiles0 + s * L::STAGE_BYTES;
                tma_load_2d(a_dst, &map_a, kb * BK, m0, full0 + 8 * s);
                tma_load_2d(a_dst + L::A_BYTES, &map_b, kb * BK + b_k0, n0 + b_row0, full0 + 8 * s);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const unsigned idesc = instr_desc(BM, BN);
            bool ok = true;
            for (int kb = 0; kb < kblocks && ok; ++kb) {
                const int s = kb % STAGES;
                const unsigned phase = (unsigned)(kb / STAGES) & 1u;
                ok = mbar_wait(full0 + 8 * s, phase, err, 2);
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const unsigned a_addr = tiles0 + s * L::STAGE_BYTES;
                const unsigned b_addr = a_addr + L::A_BYTES;
#pragma unroll
                for (int k = 0; k < BK / 16; ++k) {
                    // 16 elements of K are 32 bytes further along the swizzled row
                    mma_f16(tmem_base, smem_desc(a_addr + k * 32), smem_desc(b_addr + k * 32), idesc,
                            (kb > 0 || k > 0) ? 1u : 0u);
                }
                mma_commit(empty0 + 8 * s);               // the stage is free once these MMAs have read it
            }
            mma_commit(acc_bar);                          // the accumulator is complete
        }
    } else {
        // epilogue: warp w reads tensor-memory lanes 32 * (w % 4) .. + 31
        const int quarter = warp & 3;
        const int row = m0 + quarter * 32 + lane;
        const float ss = row_sum(rs, row, M);            // asked for while the products still run
        WeightCursor wc;
        if (ACT == ACT_WEIGHTED) wc.move(rw, row, M, n0 >> 5);
        if (mbar_wait(acc_bar, 0, err, 3)) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const float sc = rs.part ? 1.0f / sqrtf(ss * rs.inv_dim + rs.eps) : 1.f;
#pragma unroll 1
            for (int c0 = 0; c0 < BN; c0 += 32) {
                unsigned r[32];
                tmem_ld32(tmem_base + ((unsigned)(quarter * 32) << 16) + (unsigned)c0, r);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (rs.part) scale_chunk(r, sc);
                if (ACT == ACT_WEIGHTED) wc.move(rw, row, M, (n0 + c0) >> 5);
                if (row < M) store_chunk<ACT>(r, row, n0 + c0, N, mode, bias, out, ldo, wc.w);
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"((unsigned)BN)
                     : "memory");
    }
}

// ---------------------------------------------------------------------------
// The same product for wide matrices: 128 x 256 tiles, one block per SM that
// walks over tiles (consecutive blocks share a tile of W, so W comes from HBM
// once and from L2 afterwards), and TWO accumulators of 256 columns in tensor
// memory: while the epilogue warps drain one, the MMA warp fills the other, and
// the TMA warp runs ahead across tile boundaries.  A 128 x 256 tile needs
// 48 KB of operands per 128 x 256 x 64 of MMA work, 96 bytes per clock at full
// tensor rate, which four stages of shared memory can keep in flight; the
// 128 x 128 tile needs 128.
// ---------------------------------------------------------------------------
template <int STAGES>
struct WideLayout {
    static constexpr int BN = 256;
    static constexpr int A_BYTES = BM * BK * 2, B_BYTES = BN * BK * 2;
    static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
    static constexpr int TILE_BYTES = STAGES * STAGE_BYTES;
    static constexpr int BAR_BYTES = (2 * STAGES + 4) * 8 + 8;
    static constexpr int TOTAL = TILE_BYTES + BAR_BYTES + 1024;
};

template <int STAGES, int ACT>
__global__ void __launch_bounds__(THREADS, 1)
gemm_tc_wide_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b,
                    const float* __restrict__ bias, void* __restrict__ out, int mode, int M, int N, int K, int ldo,
                    const RowScale rs, const RowWeights rw, int* __restrict__ err) {
    using L = WideLayout<STAGES>;
    constexpr int BN = L::BN;
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    unsigned long long* bars = (unsigned long long*)(smem + L::TILE_BYTES);
    unsigned* tmem_holder = (unsigned*)(bars + 2 * STAGES + 4);
    const unsigned full0 = smem_u32(bars), empty0 = full0 + 8 * STAGES;
    const unsigned acc_full0 = full0 + 16 * STAGES, acc_empty0 = acc_full0 + 16;
    const unsigned tiles0 = smem_u32(smem);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int m_tiles = (M + BM - 1) / BM, n_tiles = (N + BN - 1) / BN;
    const int tiles = m_tiles * n_tiles;
    const int kblocks = (K + BK - 1) / BK;

    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) {
            mbar_init(full0 + 8 * s, 1);
            mbar_init(empty0 + 8 * s, 1);
        }
        for (int a = 0; a < 2; ++a) {
            mbar_init(acc_full0 + 8 * a, 1);
            mbar_init(acc_empty0 + 8 * a, 4);             // one arrival per epilogue warp
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;"
                     ::"r"(smem_u32(tmem_holder)), "r"(512u) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const unsigned tmem_base = *tmem_holder;

    if (warp == 0) {
        if (lane == 0) {
            int it = 0;                                   // K blocks issued so far, over all tiles
            bool ok = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                const int m0 = (t % m_tiles) * BM, n0 = (t / m_tiles) * BN;
                for (int kb = 0; kb < kblocks; ++kb, ++it) {
                    const int s = it % STAGES;
                    const unsigned phase = (unsigned)(it / STAGES) & 1u;
                    ok = mbar_wait(empty0 + 8 * s, phase ^ 1u, err, 1);
                    if (!ok) break;
                    mbar_expect_tx(full0 + 8 * s, L::STAGE_BYTES);
                    const unsigned a_dst = tiles0 + s * L::STAGE_BYTES;
                    tma_load_2d(a_dst, &map_a, kb * BK, m0, full0 + 8 * s);
                    tma_load_2d(a_dst + L::A_BYTES, &map_b, kb * BK, n0, full0 + 8 * s);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            const unsigned idesc = instr_desc(BM, BN);
            int it = 0, local = 0;
            bool ok = true;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++local) {
                const int acc = local & 1;
                const unsigned acc_phase = (unsigned)(local >> 1) & 1u;
                ok = mbar_wait(acc_empty0 + 8 * acc, acc_phase ^ 1u, err, 4);   // the epilogue has drained it
                if (!ok) break;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const unsigned tmem_acc = tmem_base + (unsigned)(acc * BN);
                for (int kb = 0; kb < kblocks; ++kb, ++it) {
                    const int s = it % STAGES;
                    const unsigned phase = (unsigned)(it / STAGES) & 1u;
                    ok = mbar_wait(full0 + 8 * s, phase, err, 2);
                    if (!ok) break;
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                    const unsigned a_addr = tiles0 + s * L::STAGE_BYTES;
                    const unsigned b_addr = a_addr + L::A_BYTES;
#pragma unroll
                    for (int k = 0; k < BK / 16; ++k)
                        mma_f16(tmem_acc, smem_desc(a_addr + k * 32), smem_desc(b_addr + k * 32), idesc,
                                (kb > 0 || k > 0) ? 1u : 0u);
                    mma_commit(empty0 + 8 * s);
                }
                mma_commit(acc_full0 + 8 * acc);
            }
        }
    } else {
        const int quarter = warp & 3;
        int local = 0;
        bool ok = true;
        for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++local) {
            const int m0 = (t % m_tiles) * BM, n0 = (t / m_tiles) * BN;
            const int acc = local & 1;
            const unsigned acc_phase = (unsigned)(local >> 1) & 1u;
            const int row = m0 + quarter * 32 + lane;
            const float ss = row_sum(rs, row, M);        // asked for while the tile's products still run
            WeightCursor wc;
            if (ACT == ACT_WEIGHTED) wc.move(rw, row, M, n0 >> 5);
            ok = mbar_wait(acc_full0 + 8 * acc, acc_phase, err, 3);
            if (!ok) break;
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const float sc = rs.part ? 1.0f / sqrtf(ss * rs.inv_dim + rs.eps) : 1.f;
#pragma unroll 1
            for (int c0 = 0; c0 < BN; c0 += 32) {
                if (n0 + c0 >= N) break;
                unsigned r[32];
                tmem_ld32(tmem_base + ((unsigned)(quarter * 32) << 16) + (unsigned)(acc * BN + c0), r);
                asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                if (rs.part) scale_chunk(r, sc);
                if (ACT == ACT_WEIGHTED) wc.move(rw, row, M, (n0 + c0) >> 5);
                if (row < M) store_chunk<ACT>(r, row, n0 + c0, N, mode, bias, out, ldo, wc.w);
            }
            // this warp has read its lanes of the accumulator: hand it back
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(acc_empty0 + 8 * acc) : "memory");
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(512u) : "memory");
    }
}

int sm_count() {
    static int n = 0;
    if (n == 0) {
        int dev = 0;
        cudaGetDevice(&dev);
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 148;
    }
    return n;
}

template <int STAGES, int ACT>
int launch_wide(const void* X, const void* W, const float* bias, void* out, int mode, int M, int N, int K, int ldo,
                const RowScale& rs, const RowWeights& rw, int* err, cudaStream_t stream) {
    using L = WideLayout<STAGES>;
    CUtensorMap ma, mb;
    if (!tensor_map(X, M, K, BM, &ma) || !tensor_map(W, N, K, L::BN, &mb)) return (int)cudaErrorInvalidValue;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(gemm_tc_wide_kernel<STAGES, ACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
        attr_set = true;
    }
    const int tiles = ((M + BM - 1) / BM) * ((N + L::BN - 1) / L::BN);
    const int blocks = tiles < sm_count() ? tiles : sm_count();
    gemm_tc_wide_kernel<STAGES, ACT><<<blocks, THREADS, L::TOTAL, stream>>>(ma, mb, bias, out, mode, M, N, K, ldo, rs, rw, err);
    return mv_launch_status();
}

template <int BN, int STAGES, int ACT>
int launch(const void* X, const void* W, const float* bias, void* out, int mode, int M, int N, int K, int ldo,
           const RowScale& rs, const RowWeights& rw, int* err, cudaStream_t stream) {
    using L = SmemLayout<BN, STAGES>;
    CUtensorMap ma, mb;
    if (!tensor_map(X, M, K, BM, &ma) || !tensor_map(W, N, K, BN, &mb)) return (int)cudaErrorInvalidValue;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(gemm_tc_kernel<BN, STAGES, ACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
        attr_set = true;
    }
    dim3 grid((N + BN - 1) / BN, (M + BM - 1) / BM);
    gemm_tc_kernel<BN, STAGES, ACT><<<grid, THREADS, L::TOTAL, stream>>>(ma, mb, bias, out, mode, M, N, K, ldo, rs, rw, err, nullptr, 0, 0);
    return mv_launch_status();
}

// The grouped form: X [M, K] sorted by group, W [w_rows, w_cols] holding every group's matrix.
template <int BN, int STAGES, int ACT>
int launch_grouped(const void* X, const void* W, const float* bias, void* out, int mode, int M, int N, int K, int ldo, int w_rows, int w_cols,
                   const int* tile_group, int b_row_step, int b_k_step, int* err, cudaStream_t stream) {
    using L = SmemLayout<BN, STAGES>;
    CUtensorMap ma, mb;
    if (!tensor_map(X, M, K, BM, &ma) || !tensor_map(W, w_rows, w_cols, BN, &mb)) return (int)cudaErrorInvalidValue;
    static bool attr_set = false;
    if (!attr_set) {
        cudaFuncSetAttribute(gemm_tc_kernel<BN, STAGES, ACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
        attr_set = true;
    }
    dim3 grid((N + BN - 1) / BN, (M + BM - 1) / BM);
    gemm_tc_kernel<BN, STAGES, ACT><<<grid, THREADS, L::TOTAL, stream>>>(ma, mb, bias, out, mode, M, N, K, ldo, RowScale{}, RowWeights{}, err,
                                                                   tile_group, b_row_step, b_k_step);
    return mv_launch_status();
}

}  // namespace

// mode: 0 store float32, 1 store bfloat16, 2 add into float32, 3 SwiGLU (W rows in groups
// of 16 gate + 16 up; out is bfloat16 [M, N/2] with row stride ldo), 4 the clamped gated activation over such rows
// (bias [N + 1]: a limit a row of W, then alpha), 5 gelu(gate) * up over such rows, 6 SwiGLU over such rows of experts
// laid end to end, gate and up times row_w[row * ld_w + expert] first (RowWeights; no bias).  ``err`` points to a
// device int that a block sets (1 producer, 2 MMA, 3 epilogue) if a wait ran out.
// Needs K a multiple of 8 and 16-byte aligned operands.  scale_part (or null): the consuming end of a
// carried norm, [M][scale_stride] with n_scale_part sums of squares a row over ``dim`` elements.
MV_API int mv_gemm_tc(const void* X, const void* W, const float* bias, void* out, int mode, int M, int N,
                      int K, int ldo, const float* scale_part, int n_scale_part, int scale_stride, int dim, float eps,
                      const float* row_w, int ld_w, int w_chunks, int w_experts, int* err, cudaStream_t stream) {
    if (M <= 0 || N <= 0) return 0;
    if (K <= 0 || K % 8 || ((uintptr_t)X & 15) || ((uintptr_t)W & 15)) return (int)cudaErrorInvalidValue;
    if (mode < 0 || mode > 6 || (mode >= 3 && (N % 32 || ldo % 2 || (mode == 4 && !bias)))) return (int)cudaErrorInvalidValue;
    if (mode == 6 && (!row_w || bias || w_chunks < 1 || w_experts < 1)) return (int)cudaErrorInvalidValue;
    const RowWeights rw = {row_w, ld_w, w_chunks, w_experts};
    if (scale_part && (n_scale_part <= 0 || n_scale_part > scale_stride || dim <= 0)) return (int)cudaErrorInvalidValue;
    RowScale rs = {};
    if (scale_part) rs = RowScale{scale_part, n_scale_part, scale_stride, 1.0f / (float)dim, eps};
#define TC_ACT(FN, A, ...) FN<__VA_ARGS__, A>(X, W, bias, out, mode, M, N, K, ldo, rs, rw, err, stream)
#define TC_GO(FN, ...)                                                                                                \
    return mode == 4   ? TC_ACT(FN, ACT_CLAMPED, __VA_ARGS__)                                                         \
           : mode == 5 ? TC_ACT(FN, ACT_GELU, __VA_ARGS__)                                                            \
           : mode == 6 ? TC_ACT(FN, ACT_WEIGHTED, __VA_ARGS__)                                                        \
                       : TC_ACT(FN, ACT_PLAIN, __VA_ARGS__)
    if (N <= 64) TC_GO(launch, 64, 4);
    // wide enough for 128 x 256 tiles to give every SM work: the persistent kernel
    const long long wide_tiles = (long long)((M + BM - 1) / BM) * ((N + 255) / 256);
    if (N >= 256 && wide_tiles >= 96) TC_GO(launch_wide, 4);
    TC_GO(launch, 128, 3);
#undef TC_GO
#undef TC_ACT
}

// The grouped product: the rows of X [M, K] are sorted by group and padded so that every tile of 128 rows belongs
// to one group (tile_group [M / 128], negative for spare tiles); W [w_rows, w_cols] holds the groups' matrices one
// below the other (b_row_step rows a group, b_k_step 0) or side by side along K (b_k_step columns a group, a
// multiple of 8; b_row_step 0); N and K are ONE group's sizes.  Modes 0 to 4 of mv_gemm_tc (no carried norm; bias, or mode 4's limits, are
// the same for every group).
// A tile's rows beyond its group's real rows hold whatever X holds there and give rows of ``out`` that nobody reads.
MV_API int mv_gemm_tc_grouped(const void* X, const void* W, const float* bias, void* out, int mode, int M, int N, int K, int ldo,
                              int w_rows, int w_cols, const int* tile_group, int b_row_step, int b_k_step, int* err,
                              cudaStream_t stream) {
    if (M <= 0 || N <= 0) return 0;
    if (K <= 0 || K % 8 || M % BM || b_k_step % 8 || !tile_group || ((uintptr_t)X & 15) || ((uintptr_t)W & 15))
        return (int)cudaErrorInvalidValue;
    if (mode > 4 || (mode >= 3 && (N % 32 || ldo % 2 || (mode == 4 && !bias)))) return (int)cudaErrorInvalidValue;
#define TC_GO(BN, S)                                                                                                       \
    return mode == 4 ? launch_grouped<BN, S, ACT_CLAMPED>(X, W, bias, out, mode, M, N, K, ldo, w_rows, w_cols, tile_group, b_row_step, \
                                                   b_k_step, err, stream)                                                  \
                     : launch_grouped<BN, S, ACT_PLAIN>(X, W, bias, out, mode, M, N, K, ldo, w_rows, w_cols, tile_group, b_row_step, \
                                                    b_k_step, err, stream)
    if (N <= 64) TC_GO(64, 4);
    TC_GO(128, 3);
#undef TC_GO
}

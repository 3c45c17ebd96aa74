// Attention over a compressed cache (see latent_attention.cu) for steps of few query tokens, bfloat16 cache, on the
// tensor cores.  All heads of a token read the same cached rows [c (rank) | r (rot)], as keys whole and as values in their
// first `rank` elements, so a token's heads are the rows of a matrix product: a block is one token, 16 heads and one share
// of the keys, and each of its 4 warps walks 16 keys in 64 by itself.  A warp's rows come into shared memory once (a
// bulk copy a row, two stages and their barriers a warp) and serve both products (mma.sync m16n8k16, float32 accumulation).
// Every warp keeps a running maximum, a denominator and an output of its own over the keys it has seen; they are put
// together at the end, the sink with them.
//
// The queries (with W_uk folded in) and the softmax weights are 32-bit numbers: each enters its product as two bfloat16
// numbers, the rounded value and what the rounding left, so scores and sums carry them to 16 bits of mantissa against the
// cache's 8.  Scores, maxima, denominators and weights are 32-bit.
#include "tc_common.cuh"

namespace {

constexpr int HT = 16;          // heads a block
constexpr int NW = 4;           // warps
constexpr int WK = 16;          // keys a warp and stage
constexpr int LK = NW * WK;     // keys of the block's warps together: shares are whole multiples
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void bulk_copy(unsigned dst, const void* src, unsigned bytes, unsigned bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, "
                 "{%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], const void* smem) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], const void* smem) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s) : "memory");
}
__device__ __forceinline__ unsigned bits(const __nv_bfloat162& v) { return *reinterpret_cast<const unsigned*>(&v); }

// row pitch of the tiles in elements: whole steps of 16, and 16 bytes more so that ldmatrix meets no bank twice
__host__ __device__ __forceinline__ int row_pitch(int w) { return (w + 15) / 16 * 16 + 8; }

// RM: output columns a block at most (a multiple of 16), FULL: exactly; blockIdx.y = head tile * column groups + column group.
template <int RM, bool FULL>
__global__ void __launch_bounds__(NW * 32)
latent_attention_decode_kernel(const float* __restrict__ qa, const __nv_bfloat16* __restrict__ pool, long long page_stride,
                               const int* __restrict__ page_table, int table_stride, int page_shift,
                               const int* __restrict__ positions, const int* __restrict__ seq_of,
                               const float* __restrict__ sinks, float* __restrict__ out, int nh, int rank, int rot,
                               float scale, int window, int splits, int col_groups, float* __restrict__ part_o,
                               float* __restrict__ part_ml, int* __restrict__ err) {
    mv_pdl_begin();
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int w = rank + rot, pitch = row_pitch(w), w16 = pitch - 8;
    __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(smem_raw);      // [NW][2][WK][pitch]
    __nv_bfloat16* qh = ks + 2 * LK * pitch;                             // [HT][pitch]: the rounded queries
    __nv_bfloat16* ql = qh + HT * pitch;                                 // [HT][pitch]: what the rounding left
    __shared__ float m_s[NW][HT], l_s[NW][HT];
    __shared__ __align__(8) unsigned long long bars[NW][2];

    const int n = blockIdx.x, split = blockIdx.z;
    const int cg = blockIdx.y % col_groups, h0 = blockIdx.y / col_groups * HT;
    const int col0 = cg * RM, cols = min(RM, rank - col0);
    const int heads = min(HT, nh - h0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = positions[n];
    const int* table = page_table + (size_t)seq_of[n] * table_stride;
    const int page_mask = (1 << page_shift) - 1;

    int j_lo = window > 0 ? max(0, pos - window + 1) : 0, j_hi = pos;
    if (splits > 1) {                                                   // this block's share: whole tiles
        const int per = ((pos - j_lo + splits) / splits + LK - 1) / LK * LK;
        j_lo += split * per;
        j_hi = min(pos, j_lo + per - 1);
        if (j_lo > j_hi) {                                              // a share without keys (never the first)
            if (cg == 0 && threadIdx.x < heads) {
                const size_t at = ((size_t)n * nh + h0 + threadIdx.x) * splits + split;
                part_ml[2 * at] = -INFINITY;
                part_ml[2 * at + 1] = 0.f;
            }
            return;
        }
    }

    __nv_bfloat16* mine = ks + (size_t)warp * 2 * WK * pitch;            // this warp's two stages
    const unsigned bar0 = smem_u32(&bars[warp][0]), mine0 = smem_u32(mine);
    const unsigned row_bytes = (unsigned)w * 2;
    // a lane copies one of the warp's 16 rows from key j0 on (rows past the end repeat the last one)
    auto load_rows = [&](int j0, int stage) {
        if (lane == 0) mbar_expect_tx(bar0 + 8 * stage, WK * row_bytes);
        __syncwarp();
        if (lane < WK) {
            const int j = min(j0 + lane, j_hi);
            bulk_copy(mine0 + (unsigned)((stage * WK + lane) * pitch * 2),
                      pool + (size_t)mv_read_page(table[j >> page_shift]) * page_stride + (size_t)(j & page_mask) * w, row_bytes,
                      bar0 + 8 * stage);
        }
    };
    if (lane == 0) {
        mbar_init(bar0, 1);
        mbar_init(bar0 + 8, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncwarp();
    const int first = j_lo + warp * WK;                                 // this warp's keys: first, first + LK, ...
    const int n_iter = first <= j_hi ? (j_hi - first) / LK + 1 : 0;
    if (n_iter > 0) load_rows(first, 0);
    if (n_iter > 1) load_rows(first + LK, 1);
    if (w16 > w)                                                        // the columns that fill up the last step of 16
        for (int e = lane; e < 2 * WK * 8; e += 32) mine[(size_t)(e >> 3) * pitch + w + (e & 7)] = __float2bfloat16(0.f);
    if (w16 > w)
        for (int e = threadIdx.x; e < 2 * HT * 8; e += NW * 32) qh[(size_t)(e >> 3) * pitch + w + (e & 7)] = __float2bfloat16(0.f);
    const float4* q4 = reinterpret_cast<const float4*>(qa + ((size_t)n * nh + h0) * w);     // the heads' rows lie together
    const int per_row = w >> 2, all_q = HT * per_row;
    for (int e0 = threadIdx.x; e0 < all_q; e0 += 4 * NW * 32) {
        float4 v[4];                                                    // four loads on their way at a time
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int e = e0 + u * NW * 32;
            v[u] = e < heads * per_row ? q4[e] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int e = e0 + u * NW * 32;
            if (e < all_q) {
                const int at = e / per_row * pitch + e % per_row * 4;
                const __nv_bfloat162 a = __floats2bfloat162_rn(v[u].x, v[u].y), b = __floats2bfloat162_rn(v[u].z, v[u].w);
                *reinterpret_cast<uint2*>(qh + at) = make_uint2(bits(a), bits(b));
                *reinterpret_cast<uint2*>(ql + at) =
                    make_uint2(bits(__floats2bfloat162_rn(v[u].x - __low2float(a), v[u].y - __high2float(a))),
                               bits(__floats2bfloat162_rn(v[u].z - __low2float(b), v[u].w - __high2float(b))));
            }
        }
    }

    float oacc[RM / 8][4];
#pragma unroll
    for (int j = 0; j < RM / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) oacc[j][e] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;           // rows lane / 4 and lane / 4 + 8; l: this lane's share
    const int t4 = lane & 3;
    const float sc = scale * LOG2E;
    const __nv_bfloat16* qh_at = qh + (lane & 15) * pitch + (lane >> 4) * 8;
    const __nv_bfloat16* ql_at = ql + (lane & 15) * pitch + (lane >> 4) * 8;
    const int k_at = ((lane & 7) + ((lane >> 4) & 1) * 8) * pitch + ((lane >> 3) & 1) * 8;
    const int v_at = ((lane & 7) + ((lane >> 3) & 1) * 8) * pitch + col0 + (lane >> 4) * 8;

    __syncthreads();                                                    // the queries are there
    for (int it = 0; it < n_iter; ++it) {
        const int j0 = first + it * LK, stage = it & 1;
        const bool ok = mbar_wait(bar0 + 8 * stage, (unsigned)(it >> 1) & 1u, err, 51);
        if (!__all_sync(0xffffffffu, ok)) {
            if (it + 1 < n_iter) mbar_wait(bar0 + 8 * (stage ^ 1), (unsigned)((it + 1) >> 1) & 1u, err, 51);   // its other copies
            break;
        }
        const __nv_bfloat16* kt = mine + (size_t)stage * WK * pitch;
        {
            float s[2][4] = {}, sl[2][4] = {};                          // the rounded queries' scores, the remainders'
#pragma unroll 4
            for (int kk = 0; kk < w16; kk += 16) {
                unsigned ah[4], al[4], b[4];
                ldmatrix_x4(ah, qh_at + kk);
                ldmatrix_x4(al, ql_at + kk);
                ldmatrix_x4(b, kt + k_at + kk);
                mma_bf16(s[0], ah, b[0], b[1]);
                mma_bf16(s[1], ah, b[2], b[3]);
                mma_bf16(sl[0], al, b[0], b[1]);
                mma_bf16(sl[1], al, b[2], b[3]);
            }
            float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const bool seen = j0 + t * 8 + 2 * t4 + e <= j_hi;
                    s[t][e] = seen ? (s[t][e] + sl[t][e]) * sc : -INFINITY;                // in units of log 2
                    s[t][e + 2] = seen ? (s[t][e + 2] + sl[t][e + 2]) * sc : -INFINITY;
                    mx0 = fmaxf(mx0, s[t][e]);
                    mx1 = fmaxf(mx1, s[t][e + 2]);
                }
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
            // (the first of the 16 keys is seen, so both maxima are finite)
            const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);
            const float c0 = exp2f(m0 - mn0), c1 = exp2f(m1 - mn1);
            m0 = mn0;
            m1 = mn1;
            float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    s[t][e] = exp2f(s[t][e] - mn0);
                    s[t][e + 2] = exp2f(s[t][e + 2] - mn1);
                    sum0 += s[t][e];
                    sum1 += s[t][e + 2];
                }
            l0 = l0 * c0 + sum0;
            l1 = l1 * c1 + sum1;
            unsigned ph[4], pl[4];
#pragma unroll
            for (int f = 0; f < 4; ++f) {
                const float x = s[f >> 1][(f & 1) * 2], y = s[f >> 1][(f & 1) * 2 + 1];
                const __nv_bfloat162 hv = __floats2bfloat162_rn(x, y);
                ph[f] = bits(hv);
                pl[f] = bits(__floats2bfloat162_rn(x - __low2float(hv), y - __high2float(hv)));
            }
            if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {      // a maximum has moved (rare after the first keys)
#pragma unroll
                for (int j = 0; j < RM / 8; ++j) {
                    oacc[j][0] *= c0; oacc[j][1] *= c0;
                    oacc[j][2] *= c1; oacc[j][3] *= c1;
                }
            }
#pragma unroll
            for (int dj = 0; dj < RM / 16; ++dj) {
                if (FULL || dj * 16 < cols) {
                    unsigned vb[4];
                    ldmatrix_x4_trans(vb, kt + v_at + dj * 16);
                    mma_bf16(oacc[2 * dj], ph, vb[0], vb[1]);
                    mma_bf16(oacc[2 * dj + 1], ph, vb[2], vb[3]);
                    mma_bf16(oacc[2 * dj], pl, vb[0], vb[1]);
                    mma_bf16(oacc[2 * dj + 1], pl, vb[2], vb[3]);
                }
            }
        }
        __syncwarp();                                                   // every lane has read the stage
        if (it + 2 < n_iter) load_rows(j0 + 2 * LK, stage);
    }

    // the warps' maxima, denominators and outputs together
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    const int g = lane >> 2;
    if (t4 == 0) {
        m_s[warp][g] = m0; l_s[warp][g] = l0;
        m_s[warp][g + 8] = m1; l_s[warp][g + 8] = l1;
    }
    __syncthreads();                                                    // (no copy is in flight any more)
    float* os = reinterpret_cast<float*>(smem_raw);                      // [NW][HT][op]: where the tiles were
    const int op = (cols + 7) / 8 * 8 + 8;                               // (op <= pitch: it fits)
    const bool with_sink = sinks && split == 0;
    auto top_of = [&](int row) {
        float M = with_sink && row < heads ? sinks[h0 + row] * LOG2E : -INFINITY;
        for (int k = 0; k < NW; ++k) M = fmaxf(M, m_s[k][row]);
        return M;
    };
    {
        const float f0 = exp2f(m0 - top_of(g)), f1 = exp2f(m1 - top_of(g + 8));   // (warp 0 has seen a key: the tops are finite)
        float* o0 = os + (size_t)(warp * HT + g) * op + 2 * t4;
        float* o1 = o0 + (size_t)8 * op;
#pragma unroll
        for (int j = 0; j < RM / 8; ++j) {
            if (FULL || j * 8 < cols) {
                *reinterpret_cast<float2*>(o0 + j * 8) = make_float2(oacc[j][0] * f0, oacc[j][1] * f0);
                *reinterpret_cast<float2*>(o1 + j * 8) = make_float2(oacc[j][2] * f1, oacc[j][3] * f1);
            }
        }
    }
    __syncthreads();
    for (int r = warp; r < heads; r += NW) {
        const float M = top_of(r);
        float L = with_sink ? exp2f(sinks[h0 + r] * LOG2E - M) : 0.f;
        for (int k = 0; k < NW; ++k) L += l_s[k][r] * exp2f(m_s[k][r] - M);
        const size_t row = (size_t)n * nh + h0 + r;
        const float inv = splits > 1 ? 1.f : 1.0f / L;
        float* dst = (splits > 1 ? part_o + (row * splits + split) * rank : out + row * rank) + col0;
        for (int c = lane; c < cols; c += 32) {
            float v = 0.f;
#pragma unroll
            for (int k = 0; k < NW; ++k) v += os[(size_t)(k * HT + r) * op + c];
            dst[c] = v * inv;
        }
        if (splits > 1 && cg == 0 && lane == 0) {
            part_ml[2 * (row * splits + split)] = M / LOG2E;             // (the shares meet in natural units)
            part_ml[2 * (row * splits + split) + 1] = L;
        }
    }
}

// The shares of one (token, head) put together: out = sum_z acc_z exp(m_z - M) / sum_z l_z exp(m_z - M), M = max m_z;
// a share without keys (m = -inf) has written nothing else.
__global__ void __launch_bounds__(128)
latent_decode_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, float* __restrict__ out,
                           int rank, int splits) {
    mv_pdl_begin();
    __shared__ float f[32];
    const size_t at = (size_t)blockIdx.x * splits;
    if (threadIdx.x < 32) {
        const int z = threadIdx.x;
        const float m = z < splits ? part_ml[2 * (at + z)] : -INFINITY;
        const float M = mv_warp_max(m);
        const float e = m == -INFINITY ? 0.f : expf(m - M);
        const float L = mv_warp_sum(z < splits ? part_ml[2 * (at + z) + 1] * e : 0.f);
        f[z] = e / L;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < rank; c += blockDim.x) {
        float a = 0.f;
        for (int z = 0; z < splits; ++z)
            if (f[z] != 0.f) a = fmaf(part_o[(at + z) * rank + c], f[z], a);
        out[(size_t)blockIdx.x * rank + c] = a;
    }
}

template <int RM, bool FULL>
int launch(const float* qa, const void* pool, long long page_stride, const int* page_table, int table_stride, int shift,
           const int* positions, const int* seq_of, const float* sinks, float* out, int N, int nh, int rank, int rot, float scale,
           int window, int splits, float* part_o, float* part_ml, int* err, cudaStream_t stream) {
    const int pitch = row_pitch(rank + rot);
    const size_t smem = (size_t)(2 * LK + 2 * HT) * pitch * sizeof(__nv_bfloat16);
    const cudaError_t e = cudaFuncSetAttribute(latent_attention_decode_kernel<RM, FULL>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    const int col_groups = (rank + RM - 1) / RM;
    const dim3 grid(N, (nh + HT - 1) / HT * col_groups, splits);
    mv_launch(latent_attention_decode_kernel<RM, FULL>, grid, NW * 32, smem, stream, qa, (const __nv_bfloat16*)pool, page_stride,
              page_table, table_stride, shift, positions, seq_of, sinks, out, nh, rank, rot, scale, window, splits, col_groups,
              part_o, part_ml, err);
    return mv_launch_status();
}

}  // namespace

MV_GUARD_SETTER(latent_attention_decode)

// qa [N, nh, rank + rot] and out [N, nh, rank], 32-bit; pool: pages of [row][rank + rot] bfloat16, rows of whole 16-byte
// pieces (rank and rot multiples of 8); sinks [nh] or null.  splits > 1 (at most 32): every (token, head tile) is that many
// blocks, each over its share of the keys, and a second kernel puts the shares together; part_o [N, nh, splits, rank]
// and part_ml [N, nh, splits, 2] are their scratch.  ``err``: a device int that a wait which ran out sets.
MV_API int mv_latent_attention_decode(const float* qa, const void* pool, long long page_stride, const int* page_table,
                                      int table_stride, int page_size, const int* positions, const int* seq_of,
                                      const float* sinks, float* out, int N, int nh, int rank, int rot, float scale, int window,
                                      int splits, float* part_o, float* part_ml, int* err, cudaStream_t stream) {
    if (N <= 0) return 0;
    if (rank < 8 || rank % 8 || rot < 0 || rot % 8 || row_pitch(rank + rot) > 688 || page_size < 1 || (page_size & (page_size - 1)) ||
        window < 0 || splits < 1 || splits > 32 || (splits > 1 && (!part_o || !part_ml)) || page_stride % 8 || ((uintptr_t)pool & 15))
        return (int)cudaErrorInvalidValue;
    int shift = 0;
    while ((1 << shift) < page_size) ++shift;
    int e;
#define LD_GO(RM)                                                                                                          \
    e = rank % RM == 0 ? launch<RM, true>(qa, pool, page_stride, page_table, table_stride, shift, positions, seq_of, sinks, out, N, \
                                          nh, rank, rot, scale, window, splits, part_o, part_ml, err, stream)             \
                       : launch<RM, false>(qa, pool, page_stride, page_table, table_stride, shift, positions, seq_of, sinks, out, \
                                           N, nh, rank, rot, scale, window, splits, part_o, part_ml, err, stream)
    if (rank <= 64) LD_GO(64);
    else if (rank <= 128) LD_GO(128);
    else LD_GO(256);
#undef LD_GO
    if (e || splits == 1) return e;
    mv_launch(latent_decode_merge_kernel, N * nh, 128, 0, stream, (const float*)part_o, (const float*)part_ml, out, rank, splits);
    return mv_launch_status();
}

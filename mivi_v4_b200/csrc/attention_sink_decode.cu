// Grouped-query softmax attention over the paged cache (see attention_sink.cu for the layer's variations) for steps of few
// query tokens, bfloat16, on the tensor cores.  The query heads of a kv head read the same keys and values, so they are the
// rows of a matrix product: a block is one token, one kv head (up to 16 of its query heads) and one share of the keys, and
// each of its 4 warps walks 16 keys in 64 by itself.  A warp's key and value rows come into shared memory once (cp.async,
// a ring of stages a warp) and serve all rows of both products (mma.sync m16n8k16, float32 accumulation).  Every warp keeps
// a running maximum, a denominator and an output of its own over the keys it has seen; they are put together at the end,
// the sink with them; shares are put together by a second kernel.
//
// Scores are scaled, capped, and given the distance table's number in float32; a softmax weight enters the second product
// as two bfloat16 numbers, the rounded weight and what the rounding left (16 bits of its mantissa).  Where a kv head has at
// most 8 query heads (PACK), rows 8 to 15 of the tile are free: they carry the remainders of rows 0 to 7, so one product
// does for both parts.
//
// Of the variations it has: keys and values of different sizes, a cap, a window, a chunked mask, a sink, a distance table.
#include "common.cuh"

namespace {

constexpr int HT = 16;          // heads a block
constexpr int NW = 4;           // warps
constexpr int WK = 16;          // keys a warp and stage
constexpr int LK = NW * WK;     // keys of the block's warps together: shares are whole multiples
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
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
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ unsigned bits(const __nv_bfloat162& v) { return *reinterpret_cast<const unsigned*>(&v); }

struct Shape {
    int nh, nkv, dk, dv, page_shift, table_stride, window, chunk, tiles, splits, dist_len;
    long long page_stride;
    float scale, cap;
};

// DVM: value elements at most (a multiple of 16); dk, dv: multiples of 16.  grid: (token, kv head * tiles + tile, share).
template <int DVM, int STAGES, bool PACK>
__global__ void __launch_bounds__(NW * 32)
attention_sink_decode_kernel(const __nv_bfloat16* __restrict__ q, const __nv_bfloat16* __restrict__ pool,
                             const int* __restrict__ page_table, const int* __restrict__ positions,
                             const int* __restrict__ seq_of, const float* __restrict__ sinks, const float* __restrict__ dist,
                             __nv_bfloat16* __restrict__ o, const Shape S, float* __restrict__ part_o,
                             float* __restrict__ part_ml) {
    mv_pdl_begin();
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int dk = S.dk, dv = S.dv, pk = dk + 8, pv = dv + 8;            // pitches: ldmatrix meets no bank twice
    __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(smem_raw);    // [NW][STAGES][WK][pk], then [WK][pv] a stage
    __nv_bfloat16* qs = ring + (size_t)NW * STAGES * WK * (pk + pv);     // [HT][pk]
    __shared__ float m_s[NW][HT], l_s[NW][HT];

    const int n = blockIdx.x, split = blockIdx.z, splits = S.splits;
    const int g = blockIdx.y / S.tiles, G = S.nh / S.nkv;
    const int h0 = g * G + (blockIdx.y - g * S.tiles) * HT;              // the tile's first query head
    const int heads = min(HT, (g + 1) * G - h0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = positions[n];
    const int* table = page_table + (size_t)seq_of[n] * S.table_stride;
    const int page_mask = (1 << S.page_shift) - 1;
    const size_t v_base = (size_t)S.nkv * (page_mask + 1) * dk;

    int j_lo = S.chunk > 0 ? pos - pos % S.chunk : (S.window > 0 ? max(0, pos - S.window + 1) : 0), j_hi = pos;
    if (splits > 1) {                                                   // this block's share: whole tiles
        const int per = ((pos - j_lo + splits) / splits + LK - 1) / LK * LK;
        j_lo += split * per;
        j_hi = min(pos, j_lo + per - 1);
        if (j_lo > j_hi) {                                              // a share without keys (never the first)
            if (threadIdx.x < heads) {
                const size_t at = ((size_t)n * S.nh + h0 + threadIdx.x) * splits + split;
                part_ml[2 * at] = -INFINITY;
                part_ml[2 * at + 1] = 0.f;
            }
            return;
        }
    }

    __nv_bfloat16* mine = ring + (size_t)warp * STAGES * WK * (pk + pv);
    const int first = j_lo + warp * WK;                                 // this warp's keys: first, first + LK, ...
    const int n_iter = first <= j_hi ? (j_hi - first) / LK + 1 : 0;
    // a stage's 16 key rows and 16 value rows, eight lanes a row (rows past the end repeat the last one)
    auto load_rows = [&](int it) {
        if (it < n_iter) {
            const int j = min(first + it * LK + (lane & 15), j_hi);
            const unsigned long long row =
                (unsigned long long)(pool + (size_t)mv_read_page(table[j >> S.page_shift]) * S.page_stride);
            const int in_page = j & page_mask;
            __nv_bfloat16* kt = mine + (size_t)(it % STAGES) * WK * (pk + pv);
            __nv_bfloat16* vt = kt + WK * pk;
#pragma unroll
            for (int r0 = 0; r0 < WK; r0 += 4) {
                const int r = r0 + (lane >> 3);
                const __nv_bfloat16* page = (const __nv_bfloat16*)__shfl_sync(0xffffffffu, row, r);
                const size_t at = (size_t)g * (page_mask + 1) + __shfl_sync(0xffffffffu, in_page, r);
                for (int c = lane & 7; c < (dk >> 3); c += 8) cp_async16(kt + r * pk + c * 8, page + at * dk + c * 8);
                for (int c = lane & 7; c < (dv >> 3); c += 8) cp_async16(vt + r * pv + c * 8, page + v_base + at * dv + c * 8);
            }
        }
        cp_async_commit();
    };
#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) load_rows(s);
    for (int e = threadIdx.x; e < HT * (dk >> 3); e += NW * 32) {       // the queries, zero where the tile has no head
        const int r = e / (dk >> 3), c = e - r * (dk >> 3);
        *reinterpret_cast<uint4*>(qs + r * pk + c * 8) =
            r < heads ? *reinterpret_cast<const uint4*>(q + ((size_t)n * S.nh + h0 + r) * dk + c * 8) : make_uint4(0, 0, 0, 0);
    }

    float oacc[DVM / 8][4];
#pragma unroll
    for (int j = 0; j < DVM / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) oacc[j][e] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;           // rows lane / 4 and lane / 4 + 8; l: this lane's share
    const int t4 = lane & 3, gq = lane >> 2;
    const float cap_l = S.cap * LOG2E, scale_l = S.cap > 0.f ? 2.0f * LOG2E * S.scale / S.cap : S.scale * LOG2E;
    const float* d0 = dist ? dist + (size_t)(h0 + min(gq, heads - 1)) * S.dist_len : nullptr;
    const float* d1 = dist ? dist + (size_t)(h0 + min(gq + 8, heads - 1)) * S.dist_len : nullptr;
    const float far0 = dist ? d0[S.dist_len - 1] : 0.f, far1 = dist ? d1[S.dist_len - 1] : 0.f;
    auto score = [&](float x, float add) {                              // in units of log 2
        // a capped score: cap tanh(y), y = scale x / cap, as cap - 2 cap / (1 + e^(2y)) (within 1e-6 of the cap's size)
        const float bias = add * LOG2E;
        return S.cap > 0.f ? fmaf(-2.0f * cap_l, rcp(1.0f + ex2(x * scale_l)), cap_l + bias) : fmaf(x, scale_l, bias);
    };
    const __nv_bfloat16* q_at = qs + (lane & 15) * pk + (lane >> 4) * 8;
    const int k_at = ((lane & 7) + ((lane >> 4) & 1) * 8) * pk + ((lane >> 3) & 1) * 8;
    const int v_at = ((lane & 7) + ((lane >> 3) & 1) * 8) * pv + (lane >> 4) * 8;

    __syncthreads();                                                    // the queries are there
    for (int it = 0; it < n_iter; ++it) {
        cp_async_wait<STAGES - 2>();
        __syncwarp();                                                   // the stage is there; the one before it is read
        load_rows(it + STAGES - 1);
        const int j0 = first + it * LK;
        const __nv_bfloat16* kt = mine + (size_t)(it % STAGES) * WK * (pk + pv);
        const __nv_bfloat16* vt = kt + WK * pk;
        // what the distance table adds to a lane's scores: asked for before the product
        const bool near = dist && pos - (j0 + WK - 1) < S.dist_len - 1;
        float add0[4], add1[4];
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const int back = pos - (j0 + (t >> 1) * 8 + 2 * t4 + (t & 1));
            add0[t] = near ? d0[min(max(back, 0), S.dist_len - 1)] : far0;
            if (!PACK) add1[t] = near ? d1[min(max(back, 0), S.dist_len - 1)] : far1;
        }
        float s[2][4] = {};
#pragma unroll 4
        for (int kk = 0; kk < dk; kk += 16) {
            unsigned a[4], b[4];
            ldmatrix_x4(a, q_at + kk);
            ldmatrix_x4(b, kt + k_at + kk);
            mma_bf16(s[0], a, b[0], b[1]);
            mma_bf16(s[1], a, b[2], b[3]);
        }
        float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const bool seen = j0 + (t >> 1) * 8 + 2 * t4 + (t & 1) <= j_hi;
            float& x = s[t >> 1][t & 1];
            x = seen ? score(x, add0[t]) : -INFINITY;
            mx0 = fmaxf(mx0, x);
            if (!PACK) {
                float& y = s[t >> 1][2 + (t & 1)];
                y = seen ? score(y, add1[t]) : -INFINITY;
                mx1 = fmaxf(mx1, y);
            }
        }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        // (the first of the 16 keys is seen, so the maxima are finite)
        const float mn0 = fmaxf(m0, mx0), c0 = ex2(m0 - mn0);
        m0 = mn0;
        float c1 = c0;
        if (!PACK) {
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
            const float mn1 = fmaxf(m1, mx1);
            c1 = ex2(m1 - mn1);
            m1 = mn1;
        }
        unsigned ph[4], pl[4];
        float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            const float x = ex2(s[t][0] - m0), y = ex2(s[t][1] - m0);
            sum0 += x + y;
            const __nv_bfloat162 hv = __floats2bfloat162_rn(x, y);
            const unsigned rest = bits(__floats2bfloat162_rn(x - __low2float(hv), y - __high2float(hv)));
            ph[2 * t] = bits(hv);
            if (PACK) {
                ph[2 * t + 1] = rest;                                   // rows 8 to 15: the remainders
            } else {
                pl[2 * t] = rest;
                const float x1 = ex2(s[t][2] - m1), y1 = ex2(s[t][3] - m1);
                sum1 += x1 + y1;
                const __nv_bfloat162 h1 = __floats2bfloat162_rn(x1, y1);
                ph[2 * t + 1] = bits(h1);
                pl[2 * t + 1] = bits(__floats2bfloat162_rn(x1 - __low2float(h1), y1 - __high2float(h1)));
            }
        }
        l0 = l0 * c0 + sum0;
        if (!PACK) l1 = l1 * c1 + sum1;
        if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {          // a maximum has moved (rare after the first keys)
#pragma unroll
            for (int j = 0; j < DVM / 8; ++j) {
                oacc[j][0] *= c0; oacc[j][1] *= c0;
                oacc[j][2] *= c1; oacc[j][3] *= c1;
            }
        }
#pragma unroll
        for (int dj = 0; dj < DVM / 16; ++dj) {
            if (dj * 16 < dv) {
                unsigned vb[4];
                ldmatrix_x4_trans(vb, vt + v_at + dj * 16);
                mma_bf16(oacc[2 * dj], ph, vb[0], vb[1]);
                mma_bf16(oacc[2 * dj + 1], ph, vb[2], vb[3]);
                if (!PACK) {
                    mma_bf16(oacc[2 * dj], pl, vb[0], vb[1]);
                    mma_bf16(oacc[2 * dj + 1], pl, vb[2], vb[3]);
                }
            }
        }
    }

    // the warps' maxima, denominators and outputs together
    cp_async_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
    l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    if (t4 == 0) {
        m_s[warp][gq] = m0; l_s[warp][gq] = l0;
        m_s[warp][gq + 8] = m1; l_s[warp][gq + 8] = l1;
    }
    __syncthreads();                                                    // (no copy is in flight, no stage is read any more)
    float* os = reinterpret_cast<float*>(smem_raw);                     // [NW][HT][op]: where the stages were
    const int op = dv + 8;
    const bool with_sink = sinks && split == 0;
    auto top_of = [&](int row) {
        float M = with_sink && row < heads ? sinks[h0 + row] * LOG2E : -INFINITY;
        for (int k = 0; k < NW; ++k) M = fmaxf(M, m_s[k][row]);
        return M;
    };
    {
        const float f0 = ex2(m0 - top_of(gq));                        // (warp 0 has seen a key: the tops are finite)
        const float f1 = PACK ? 0.f : ex2(m1 - top_of(gq + 8));
        float* o0 = os + (size_t)(warp * HT + gq) * op + 2 * t4;
        float* o1 = o0 + (size_t)8 * op;
#pragma unroll
        for (int j = 0; j < DVM / 8; ++j) {
            if (j * 8 < dv) {
                if (PACK) {
                    *reinterpret_cast<float2*>(o0 + j * 8) = make_float2((oacc[j][0] + oacc[j][2]) * f0, (oacc[j][1] + oacc[j][3]) * f0);
                } else {
                    *reinterpret_cast<float2*>(o0 + j * 8) = make_float2(oacc[j][0] * f0, oacc[j][1] * f0);
                    *reinterpret_cast<float2*>(o1 + j * 8) = make_float2(oacc[j][2] * f1, oacc[j][3] * f1);
                }
            }
        }
    }
    __syncthreads();
    for (int r = warp; r < heads; r += NW) {
        const float M = top_of(r);
        float L = with_sink ? ex2(sinks[h0 + r] * LOG2E - M) : 0.f;
        for (int k = 0; k < NW; ++k) L += l_s[k][r] * ex2(m_s[k][r] - M);
        const size_t row = (size_t)n * S.nh + h0 + r;
        const float inv = 1.0f / L;
        for (int c = lane; c < dv; c += 32) {
            float v = 0.f;
#pragma unroll
            for (int k = 0; k < NW; ++k) v += os[(size_t)(k * HT + r) * op + c];
            if (splits > 1) part_o[(row * splits + split) * dv + c] = v;
            else o[row * dv + c] = __float2bfloat16_rn(v * inv);
        }
        if (splits > 1 && lane == 0) {
            part_ml[2 * (row * splits + split)] = M;                    // (in units of log 2)
            part_ml[2 * (row * splits + split) + 1] = L;
        }
    }
}

// The shares of one (token, head) put together: out = sum_z acc_z 2^(m_z - M) / sum_z l_z 2^(m_z - M), M = max m_z;
// a share without keys (m = -inf) has written nothing else.
__global__ void __launch_bounds__(64)
sink_decode_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, __nv_bfloat16* __restrict__ out,
                         int dv, int splits) {
    mv_pdl_begin();
    __shared__ float f[32];
    const size_t at = (size_t)blockIdx.x * splits;
    if (threadIdx.x < 32) {
        const int z = threadIdx.x;
        const float m = z < splits ? part_ml[2 * (at + z)] : -INFINITY;
        const float M = mv_warp_max(m);
        const float e = m == -INFINITY ? 0.f : exp2f(m - M);
        const float L = mv_warp_sum(z < splits ? part_ml[2 * (at + z) + 1] * e : 0.f);
        f[z] = e / L;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < dv; c += blockDim.x) {
        float a = 0.f;
        for (int z = 0; z < splits; ++z)
            if (f[z] != 0.f) a = fmaf(part_o[(at + z) * dv + c], f[z], a);
        out[(size_t)blockIdx.x * dv + c] = __float2bfloat16_rn(a);
    }
}

template <int DVM, int STAGES, bool PACK>
int launch(const void* q, const void* pool, const int* page_table, const int* positions, const int* seq_of, const float* sinks,
           const float* dist, void* o, const Shape& S, int N, float* part_o, float* part_ml, cudaStream_t stream) {
    const size_t smem = ((size_t)NW * STAGES * WK * (S.dk + 8 + S.dv + 8) + HT * (S.dk + 8)) * sizeof(__nv_bfloat16);
    const cudaError_t e = cudaFuncSetAttribute(attention_sink_decode_kernel<DVM, STAGES, PACK>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    mv_launch(attention_sink_decode_kernel<DVM, STAGES, PACK>, dim3(N, S.nkv * S.tiles, S.splits), NW * 32, smem, stream,
              (const __nv_bfloat16*)q, (const __nv_bfloat16*)pool, page_table, positions, seq_of, sinks, dist,
              (__nv_bfloat16*)o, S, part_o, part_ml);
    return mv_launch_status();
}

}  // namespace

MV_GUARD_SETTER(attention_sink_decode)

// q [N, nh * dk], o [N, nh * dv] bfloat16; pool: pages of [kv head][row][dk] keys, then [kv head][row][dv] values, bfloat16;
// dk and dv multiples of 16 up to 256; sinks [nh] or null; dist 32-bit [nh, dist_len] or null.  splits > 1 (at most 32):
// every (token, kv head) is that many blocks, each over its share of the keys; part_o 32-bit [N, nh, splits, dv] and
// part_ml [N, nh, splits, 2] are their scratch.
MV_API int mv_attention_sink_decode(const void* q, const void* pool, long long page_stride, const int* page_table,
                                    int table_stride, int page_size, const int* positions, const int* seq_of,
                                    const float* sinks, const float* dist, int dist_len, void* o, int N, int nh, int nkv,
                                    int dk, int dv, float scale, float cap, int window, int chunk, int splits, float* part_o,
                                    float* part_ml, cudaStream_t stream) {
    if (N <= 0) return 0;
    if (nkv < 1 || nh % nkv || dk < 16 || dk % 16 || dk > 256 || dv < 16 || dv % 16 || dv > 256 || page_size < 1 ||
        (page_size & (page_size - 1)) || window < 0 || chunk < 0 || splits < 1 || splits > 32 || (splits > 1 && (!part_o || !part_ml)) ||
        (dist && dist_len < 1) || page_stride % 8 || (((uintptr_t)pool | (uintptr_t)q) & 15))
        return (int)cudaErrorInvalidValue;
    Shape S = {};
    S.nh = nh; S.nkv = nkv; S.dk = dk; S.dv = dv;
    while ((1 << S.page_shift) < page_size) ++S.page_shift;
    const int G = nh / nkv;
    S.table_stride = table_stride; S.window = window; S.chunk = chunk; S.tiles = (G + HT - 1) / HT; S.splits = splits;
    S.dist_len = dist_len; S.page_stride = page_stride; S.scale = scale; S.cap = cap;
    int e;
#define SD_GO(DVM, ST)                                                                                                    \
    e = G <= 8 ? launch<DVM, ST, true>(q, pool, page_table, positions, seq_of, sinks, dist, o, S, N, part_o, part_ml, stream) \
               : launch<DVM, ST, false>(q, pool, page_table, positions, seq_of, sinks, dist, o, S, N, part_o, part_ml, stream)
    if (dv <= 64) SD_GO(64, 3);
    else if (dv <= 128) SD_GO(128, 3);
    else SD_GO(256, 2);
#undef SD_GO
    if (e || splits == 1) return e;
    mv_launch(sink_decode_merge_kernel, N * nh, 64, 0, stream, (const float*)part_o, (const float*)part_ml, (__nv_bfloat16*)o, dv, splits);
    return mv_launch_status();
}

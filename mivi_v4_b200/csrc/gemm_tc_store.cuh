// The epilogue of the tcgen05 matrix products: one row's 32 consecutive columns of the accumulator,
// from registers to Y, in the mode asked for (0 store float32, 1 store bfloat16, 2 add into float32,
// 3 SwiGLU over columns that alternate in groups of 16 gate and 16 up values, 4 the clamped gated activation over
// such columns, ``bias`` then holding a limit a column and, after them, alpha, 5 gelu (its tanh form) of the gate times up,
// 6 SwiGLU of gate and up times a weight a row and an expert, see RowWeights).  Included inside the including file's
// own namespace.
// Mode 6: the columns are experts' gates and ups end to end, 32 * chunks of an expert; a row's weight for its expert e, w[row *
// ld + e], multiplies gate and up before the activation (the expert's input carries it).  Columns after the last expert's
// take 1.
struct RowWeights {
    const float* w;
    int ld, chunks, n_experts;
};
// A row's weight for the 32-column chunk c, kept until the next expert's columns begin: a tile mostly holds one expert's,
// and its weight is asked for before the tile's products are done.
struct WeightCursor {
    int end = 0;                   // the chunk where the held weight's expert ends
    float w = 1.f;
    __device__ __forceinline__ void move(const RowWeights& rw, int row, int M, int c) {
        if (c < end) return;
        const int e = c / rw.chunks;
        w = e < rw.n_experts && row < M ? rw.w[(size_t)row * rw.ld + e] : 1.f;
        end = e < rw.n_experts ? (e + 1) * rw.chunks : 0x7fffffff;
    }
};
// One row's 32 consecutive columns of the accumulator, from registers to Y, in the mode asked for.
// wt: mode 6's weight.
// ACT: an instance of its own for each of the modes 4, 5 and 6 (the branches would cost the other modes registers).
enum { ACT_PLAIN = 0, ACT_CLAMPED = 1, ACT_GELU = 2, ACT_WEIGHTED = 3 };
template <int ACT>
__device__ __forceinline__ void store_chunk(const unsigned (&r)[32], int row, int n_base, int N, int mode,
                                            const float* __restrict__ bias, void* __restrict__ out, int ldo,
                                            float wt) {

        constexpr bool CLAMP = ACT == ACT_CLAMPED;
        if (ACT != ACT_PLAIN || mode == 3) {
            // columns n_base .. +15 are gate, +16 .. +31 the up values of the same features
            if (n_base + 32 <= N) {
                __nv_bfloat16* dst = (__nv_bfloat16*)out + (size_t)row * ldo + (n_base >> 1);
                unsigned packed[8];
                const float limit = CLAMP ? bias[n_base] : 0.f, alpha = CLAMP ? bias[N] : 0.f;
#pragma unroll
                for (int j = 0; j < 16; j += 2) {
                    float a0 = __uint_as_float(r[j]), a1 = __uint_as_float(r[j + 1]);
                    float b0 = __uint_as_float(r[j + 16]), b1 = __uint_as_float(r[j + 17]);
                    if (ACT == ACT_WEIGHTED) { a0 *= wt; a1 *= wt; b0 *= wt; b1 *= wt; }
                    if ((ACT == ACT_PLAIN || ACT == ACT_GELU) && bias) {
                        a0 += bias[n_base + j]; a1 += bias[n_base + j + 1];
                        b0 += bias[n_base + j + 16]; b1 += bias[n_base + j + 17];
                    }
                    const __nv_bfloat162 v =
                        CLAMP ? __floats2bfloat162_rn(mv_glu_clamped(a0, b0, limit, alpha), mv_glu_clamped(a1, b1, limit, alpha))
                        : ACT == ACT_GELU ? __floats2bfloat162_rn(mv_glu_gelu_fast(a0, b0), mv_glu_gelu_fast(a1, b1))
                        : ACT == ACT_WEIGHTED ? __floats2bfloat162_rn(mv_glu_silu_fast(a0, b0), mv_glu_silu_fast(a1, b1))
                              : __floats2bfloat162_rn(mv_glu_silu(a0, b0), mv_glu_silu(a1, b1));
                    packed[j >> 1] = *reinterpret_cast<const unsigned*>(&v);
                }
                if ((((uintptr_t)dst) & 15) == 0) {
                    reinterpret_cast<uint4*>(dst)[0] = make_uint4(packed[0], packed[1], packed[2], packed[3]);
                    reinterpret_cast<uint4*>(dst)[1] = make_uint4(packed[4], packed[5], packed[6], packed[7]);
                } else {
#pragma unroll
                    for (int j = 0; j < 8; ++j) reinterpret_cast<unsigned*>(dst)[j] = packed[j];
                }
            }
        } else if (mode == 1) {
            __nv_bfloat16* dst = (__nv_bfloat16*)out + (size_t)row * ldo + n_base;
#pragma unroll
            for (int j = 0; j < 32; ++j) {
                if (n_base + j < N) {
                    float v = __uint_as_float(r[j]);
                    if (bias) v += bias[n_base + j];
                    dst[j] = __float2bfloat16_rn(v);
                }
            }
        } else {
            float* dst = (float*)out + (size_t)row * ldo + n_base;
            const bool vec = n_base + 32 <= N && (((uintptr_t)dst) & 15) == 0;
            if (vec) {
#pragma unroll
                for (int j = 0; j < 32; j += 4) {
                    float4 v = make_float4(__uint_as_float(r[j]), __uint_as_float(r[j + 1]),
                                           __uint_as_float(r[j + 2]), __uint_as_float(r[j + 3]));
                    if (bias) {
                        const float4 bb = *reinterpret_cast<const float4*>(bias + n_base + j);
                        v.x += bb.x; v.y += bb.y; v.z += bb.z; v.w += bb.w;
                    }
                    float4* p = reinterpret_cast<float4*>(dst + j);
                    if (mode == 2) {
                        // added in memory: nothing comes back, so the epilogue does not wait for a read
                        // (one add an element a product: the same sum as load, add, store)
                        asm volatile("red.global.add.v4.f32 [%0], {%1, %2, %3, %4};"
                                     ::"l"(p), "f"(v.x), "f"(v.y), "f"(v.z), "f"(v.w) : "memory");
                    } else {
                        *p = v;
                    }
                }
            } else {
#pragma unroll
                for (int j = 0; j < 32; ++j) {
                    if (n_base + j < N) {
                        float v = __uint_as_float(r[j]);
                        if (bias) v += bias[n_base + j];
                        if (mode == 2) v += dst[j];
                        dst[j] = v;
                    }
                }
            }
        }

}


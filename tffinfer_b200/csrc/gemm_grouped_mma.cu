// The grouped product of gemm_grouped.cu for bfloat16 operands on the tensor cores (mma.sync m16n8k16, float32
// accumulation): C_g[m, n] = sum_k A_g[m, k] * B_g[n, k], uniform or ragged groups, optional row map, as there.
// Tiles of 128 x 128 x 64, eight warps of 32 x 64, operands through a three-stage cp.async ring into padded shared
// memory (rows of 144 bytes: the eight rows of an ldmatrix fall into different banks), fragments by ldmatrix.
// Gated form: B_g holds the gate and up rows of a group alternating in blocks of 64 ([g0..g63 | u0..u63 | g64.. ], the
// layout of the tcgen05 products), a tile of 128 rows of B being one such pair of blocks; a warp then takes 32 gate
// rows and the 32 up rows of the same outputs, so that a thread finds act(gate) and up of an output element four
// accumulator tiles apart; C_g[m, f] = act(gate_f) * up_f has half as many columns as B_g has rows.
// Steps of few rows a group (decoded tokens: a token or two an expert, a token or eight a head) take tiles of 16 rows
// instead: the eight warps lie side by side along B's rows, so that a tile multiplies 16 rows and not 128 of which most
// are not there, and the ring is deeper (five stages, two CTAs an SM), since such a product is a pass of the weights.
// Needs K, lda, ldb and the group strides to be multiples of 8 elements and 16-byte aligned bases (the launcher
// refuses anything else and the caller takes the FMA kernel).  A row's result does not depend on the tile it is in:
// every output element adds its products in the same order of k.
#include "common.cuh"

namespace {

constexpr int MBN = 128, MBK = 64, LDS = MBK + 8, THREADS = 256;
constexpr int CHUNKS = MBK / 8;                          // 16-byte pieces of a tile row
constexpr int BIG_ROWS = 128, SMALL_ROWS = 16;           // rows of a tile
template <int BM> struct RingCfg {
    static constexpr int kStages = BM == SMALL_ROWS ? 5 : 3;
    static constexpr int kSmem = kStages * (BM + MBN) * LDS * 2;
};

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, int bytes) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// act(g) u; act 3 is g' sigmoid(slope g') (u' + 1), g' = min(g, limit), u' = u held within -limit .. limit
__device__ __forceinline__ float gate_of(float g, float u, int act, float limit, float slope) {
    if (act == 0) return g / (1.0f + expf(-g)) * u;
    if (act == 3) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g / (1.0f + expf(-slope * g)) * (u + 1.0f);
    }
    const float c = 0.7978845608028654f * (g + 0.044715f * g * g * g);
    return 0.5f * g * (1.0f + tanhf(c)) * u;
}

template <typename TCc, bool GATED, int MBM>
__global__ void __launch_bounds__(THREADS, 2)
gemm_grouped_mma_kernel(const bf16* __restrict__ A, long long lda, long long a_gs,
                        const bf16* __restrict__ B, long long ldb, long long b_gs,
                        TCc* __restrict__ C, long long ldc, long long c_gs,
                        const int* __restrict__ tile_group, const int* __restrict__ tile_row0,
                        const int* __restrict__ tile_row_end, const int* __restrict__ num_tiles,
                        const int* __restrict__ row_map, const int* __restrict__ a_rows, int M, int N, int K, int act,
                        float limit, float slope) {
    constexpr int STAGES = RingCfg<MBM>::kStages;
    constexpr bool SMALL = MBM == SMALL_ROWS;
    constexpr int MI = SMALL ? 1 : 2, NJ = SMALL ? 1 : 4;     // a warp's 16-row pieces of A and of B
    constexpr int A_LOADS = (MBM * CHUNKS + THREADS - 1) / THREADS;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* As = (bf16*)smem_raw;                               // [STAGES][MBM][LDS]
    bf16* Bs = As + STAGES * MBM * LDS;                       // [STAGES][MBN][LDS]
    pdl_launch_dependents();
    pdl_wait();
    int g, m0, m_end;
    if (tile_group != nullptr) {
        if ((int)blockIdx.y >= __ldcg(num_tiles)) return;        // the tables are a kernel's ahead: past the first-level cache
        g = __ldcg(tile_group + blockIdx.y); m0 = __ldcg(tile_row0 + blockIdx.y); m_end = __ldcg(tile_row_end + blockIdx.y);
    } else {
        g = blockIdx.z; m0 = blockIdx.y * MBM; m_end = M;
    }
    const int n0 = blockIdx.x * MBN;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int wm = SMALL ? 0 : warp >> 1, wn = SMALL ? warp : warp & 1;      // 4 x 2 warps of 32 x 64, or 8 of 16 x 16
    const bf16* Ag = A + (size_t)g * a_gs;
    const bf16* Bg = B + (size_t)g * b_gs;
    const int kt = (K + MBK - 1) / MBK;
    // where this thread's rows of A lie (row r of the sorted order is row a_rows[r] of A when there is such a table)
    long long a_off[A_LOADS];
#pragma unroll
    for (int i = 0; i < A_LOADS; ++i) {
        const int r = m0 + (tid + i * THREADS) / CHUNKS;
        a_off[i] = r < m_end ? (long long)(a_rows ? __ldcg(a_rows + r) : r) * lda : 0;
    }

    auto load_stage = [&](int s, int k0) {
#pragma unroll
        for (int i = 0; i < A_LOADS; ++i) {
            const int c = tid + i * THREADS, r = c / CHUNKS, kc = (c % CHUNKS) * 8;
            if (SMALL && r >= MBM) break;
            const bool oka = k0 + kc < K && (m0 + r < m_end);
            cp_async16(smem_addr(As + ((size_t)s * MBM + r) * LDS + kc),
                       oka ? (const void*)(Ag + a_off[i] + k0 + kc) : (const void*)Ag, oka ? 16 : 0);
        }
#pragma unroll
        for (int i = 0; i < MBN * CHUNKS / THREADS; ++i) {
            const int c = tid + i * THREADS, r = c / CHUNKS, kc = (c % CHUNKS) * 8;
            const bool okb = k0 + kc < K && (n0 + r < N);
            cp_async16(smem_addr(Bs + ((size_t)s * MBN + r) * LDS + kc),
                       okb ? (const void*)(Bg + (size_t)(n0 + r) * ldb + k0 + kc) : (const void*)Bg, okb ? 16 : 0);
        }
    };

    float acc[MI][2 * NJ][4];
#pragma unroll
    for (int i = 0; i < MI; ++i)
#pragma unroll
        for (int j = 0; j < 2 * NJ; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;

#pragma unroll
    for (int s = 0; s < STAGES - 1; ++s) {
        if (s < kt) load_stage(s, s * MBK);
        cp_commit();
    }
    for (int kb = 0; kb < kt; ++kb) {
        cp_wait<STAGES - 2>();
        __syncthreads();
        const int nk = kb + STAGES - 1;
        if (nk < kt) load_stage(nk % STAGES, nk * MBK);
        cp_commit();
        const bf16* as = As + (size_t)(kb % STAGES) * MBM * LDS;
        const bf16* bs = Bs + (size_t)(kb % STAGES) * MBN * LDS;
#pragma unroll
        for (int kk = 0; kk < MBK; kk += 16) {
            uint32_t a[MI][4], b[NJ][4];
#pragma unroll
            for (int mi = 0; mi < MI; ++mi)
                ldsm4(a[mi], smem_addr(as + (size_t)(wm * 32 + mi * 16 + (lane & 15)) * LDS + kk + (lane >> 4) * 8));
#pragma unroll
            for (int nj = 0; nj < NJ; ++nj) {
                // rows of B this warp's 16-row slice nj covers: plain 64 in a row; gated 32 gate rows, then their 32 up
                // rows (tiles of 16 rows: 16 in a row, or 8 gate rows and their 8 up rows)
                const int brow = SMALL ? (GATED ? wn * 8 + (lane >> 4) * 56 : wn * 16)
                                       : GATED ? ((nj >> 1) * 64 + wn * 32 + (nj & 1) * 16) : (wn * 64 + nj * 16);
                ldsm4(b[nj], smem_addr(bs + (size_t)(brow + (lane & 7) + (lane >> 4) * 8) * LDS + kk + ((lane >> 3) & 1) * 8));
            }
#pragma unroll
            for (int mi = 0; mi < MI; ++mi)
#pragma unroll
                for (int nj = 0; nj < NJ; ++nj) {
                    mma16816(acc[mi][2 * nj], a[mi], b[nj][0], b[nj][1]);
                    mma16816(acc[mi][2 * nj + 1], a[mi], b[nj][2], b[nj][3]);
                }
        }
    }
    cp_wait<0>();

#pragma unroll
    for (int mi = 0; mi < MI; ++mi)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int m = m0 + wm * 32 + mi * 16 + (lane >> 2) + half * 8;
            if (m >= m_end) continue;
            const long long row = row_map ? __ldcg(row_map + m) : m;
            TCc* crow = C + (size_t)g * c_gs + (size_t)row * ldc;
            if constexpr (GATED) {
#pragma unroll
                for (int t = 0; t < NJ; ++t) {
                    const int f = n0 / 2 + wn * (NJ * 8) + t * 8 + 2 * (lane & 3);
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        if (f + e < N / 2)
                            crow[f + e] = from_f32<TCc>(gate_of(acc[mi][t][half * 2 + e], acc[mi][t + NJ][half * 2 + e], act, limit, slope));
                }
            } else {
#pragma unroll
                for (int nj = 0; nj < 2 * NJ; ++nj) {
                    const int n = n0 + wn * (NJ * 16) + nj * 8 + 2 * (lane & 3);
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        if (n + e < N) {
                            float v = acc[mi][nj][half * 2 + e];
                            if (act == 2) { v = fmaxf(v, 0.f); v = v * v; }     // the square of relu behind a plain product
                            crow[n + e] = from_f32<TCc>(v);
                        }
                }
            }
        }
}

}  // namespace

// A and B bfloat16.  gated != 0: B's N rows are gate and up rows alternating in blocks of 64 and C has N / 2 columns.
// c_dt 0 = float32, 1 = bfloat16.  ``a_rows`` (ragged form; null: A is in the sorted order), ``act``, ``limit`` and ``slope``
// as for tff_gemm_grouped.  tile_rows: 128, or 16 for steps of few rows a group.  The ragged form's tiles must have been planned with it.
TFF_API int tff_gemm_grouped_mma(
    const void* A, long long lda, long long a_gs, const void* B, long long ldb, long long b_gs,
    void* C, int c_dt, long long ldc, long long c_gs,
    const int* tile_group, const int* tile_row0, const int* tile_row_end, const int* num_tiles, int max_tiles,
    const int* row_map, const int* a_rows, int groups, int M, int N, int K, int gated, int act, float limit, float slope,
    int tile_rows, cudaStream_t stream) {
    if (N <= 0 || K <= 0 || !A || !B || !C || (tile_rows != BIG_ROWS && tile_rows != SMALL_ROWS)) return TFF_ERR_BAD_ARGUMENT;
    if ((K & 7) || (lda & 7) || (ldb & 7) || (a_gs & 7) || (b_gs & 7) || ((uintptr_t)A & 15) || ((uintptr_t)B & 15) ||
        (gated && (N & 127)))
        return TFF_ERR_UNSUPPORTED;
    dim3 grid;
    if (tile_group) {
        if (!tile_row0 || !tile_row_end || !num_tiles) return TFF_ERR_BAD_ARGUMENT;
        if (max_tiles <= 0) return TFF_OK;
        grid = dim3((N + MBN - 1) / MBN, max_tiles, 1);
    } else {
        if (M <= 0 || groups <= 0) return TFF_OK;
        if (groups > 65535) return TFF_ERR_UNSUPPORTED;
        grid = dim3((N + MBN - 1) / MBN, (M + tile_rows - 1) / tile_rows, groups);
    }
    if (grid.y > 65535) return TFF_ERR_UNSUPPORTED;
#define TFF_GM(TCc, G)                                                                                              \
    do {                                                                                                            \
        if (tile_rows == SMALL_ROWS) TFF_GM_ROWS(TCc, G, SMALL_ROWS);                                               \
        TFF_GM_ROWS(TCc, G, BIG_ROWS);                                                                              \
    } while (0)
#define TFF_GM_ROWS(TCc, G, BM)                                                                                     \
    do {                                                                                                            \
        constexpr int smem = RingCfg<BM>::kSmem;                                                                    \
        cudaFuncSetAttribute(gemm_grouped_mma_kernel<TCc, G, BM>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem); \
        return tff_launch_pdl(gemm_grouped_mma_kernel<TCc, G, BM>, grid, dim3(THREADS), (size_t)smem, stream,       \
                              (const bf16*)A, lda, a_gs, (const bf16*)B, ldb, b_gs, (TCc*)C, ldc, c_gs, tile_group, \
                              tile_row0, tile_row_end, num_tiles, row_map, a_rows, M, N, K, act, limit, slope);                           \
    } while (0)
    if (c_dt == 0 && gated) TFF_GM(float, true);
    if (c_dt == 0) TFF_GM(float, false);
    if (c_dt == 1 && gated) TFF_GM(bf16, true);
    if (c_dt == 1) TFF_GM(bf16, false);
#undef TFF_GM
#undef TFF_GM_ROWS
    return TFF_ERR_BAD_ARGUMENT;
}

TFF_API int tff_gemm_grouped_mma_tile_rows(int few_rows) { return few_rows ? SMALL_ROWS : BIG_ROWS; }

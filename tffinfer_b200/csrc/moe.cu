// The small kernels around a routed feed-forward (mixture of experts); the experts' products are gemm_grouped.cu.
//
//   route    per token: z = W_r h in float32 (one warp per expert, a fixed order of additions), s = sigmoid(z) or
//            softmax(z) over all outputs (or z itself, the chosen then weighted by a softmax among themselves; z may
//            carry a bias), choice scores s + correction, optionally only the experts of the best
//            ``keep`` of ``groups`` groups of neighbours (a group's score is its best choice score), the ``top`` experts
//            of largest choice score (the lower index wins a tie), weights s, optionally renormalised to sum 1; writes
//            the pair (token, k) -> (expert, weight) and counts the pairs of every expert.  The last router outputs may
//            be identity experts (output = weight * input): their pairs get expert -1, no row in the experts' products,
//            and the combine kernel adds them from the input rows
//   plan     one block: the experts' row ranges in the sorted order, the tile table of the grouped product (tiles of
//            ``tile_rows`` rows that never span two experts), and the counters back to zero for the next call
//   table    instead of route and plan where a table gives every token id its experts (no router): one block counts the
//            experts' pairs in shared memory, lays out their rows and tiles as plan does, and gives every pair its place
//            (an atomic cursor in shared memory, as gather's), its weight 1/top, and every place its token row.  Behind
//            the router's kernel (no table) it stands for plan and gather in steps of few pairs, whose products read
//            the tokens' rows where they are
//   gather   per pair: its place among its expert's rows (an atomic cursor: the order within an expert is not fixed,
//            but a row's result does not depend on its place), row_map[place] = pair, and the expert's input row
//            x[place] = w * h[token] (weight on the input) or h[token]
//   combine  per token: residual[t] += sum_k y[t * top + k] (times the weight when it multiplies the output), in
//            the order k = 0 .. top-1
#include "common.cuh"

namespace {

// Tokens a block of moe_route_kernel takes (one warp each for the choice) and its threads: steps of many tokens share the
// reading of the router's rows, steps of few give every output a warp of its own.
constexpr int ROUTE_MANY_TOK = 4, ROUTE_MANY_THREADS = 256, ROUTE_FEW_TOK = 1, ROUTE_FEW_THREADS = 1024, ROUTE_FEW = 256;

template <typename TH, typename TW, int ROUTE_TOK, int ROUTE_THREADS>
__global__ void __launch_bounds__(ROUTE_THREADS)
moe_route_kernel(const TH* __restrict__ h, const TW* __restrict__ w_router, const float* __restrict__ bias, int T, int W, int E,
                 int top, int renormalize, int softmax_scores, const float* __restrict__ correction, int groups, int keep, int num_real,
                 int* __restrict__ pair_expert, float* __restrict__ pair_weight, int* __restrict__ counts,
                 const TW* __restrict__ row_w, float* __restrict__ row_out) {
    // A block takes ROUTE_TOK tokens: the router's rows are read once for all of them (2,048 tokens re-read a 64 KB router
    // 2,048 times otherwise), every token keeps sums of its own, and behind the products warp i does token i's choice.
    extern __shared__ float sm[];              // per token W floats (its row) and 3 E: the scores, the choice scores, groups
    pdl_launch_dependents();
    const int t0 = blockIdx.x * ROUTE_TOK, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // the weights are older than the kernels ahead: into the second-level cache while those are still at work
    if (ROUTE_TOK == 1)
        for (size_t e = (size_t)threadIdx.x * 128; e < (size_t)E * W * sizeof(TW); e += (size_t)ROUTE_THREADS * 128)
            asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(w_router) + e));
    pdl_wait();
    const int nt = min(ROUTE_TOK, T - t0);
    float* rows = sm;                          // [ROUTE_TOK][W]
    float* scores = sm + (size_t)ROUTE_TOK * W;   // [ROUTE_TOK][3 E]
    if ((W & 7) == 0 && ((size_t)h & 15) == 0) {           // eight elements a load (sixteen bytes of bfloat16)
        for (int v = threadIdx.x; v < nt * (W >> 3); v += ROUTE_THREADS) {
            const int k = v / (W >> 3), i = (v - k * (W >> 3)) << 3;
            float* dst = rows + (size_t)k * W + i;
            const TH* src = h + (size_t)(t0 + k) * W + i;
            if constexpr (sizeof(TH) == 2) {
                const uint4 raw = *reinterpret_cast<const uint4*>(src);
                const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
                const float2 a = __bfloat1622float2(p2[0]), b = __bfloat1622float2(p2[1]);
                const float2 c = __bfloat1622float2(p2[2]), d = __bfloat1622float2(p2[3]);
                *reinterpret_cast<float4*>(dst) = make_float4(a.x, a.y, b.x, b.y);
                *reinterpret_cast<float4*>(dst + 4) = make_float4(c.x, c.y, d.x, d.y);
            } else {
                *reinterpret_cast<float4*>(dst) = *reinterpret_cast<const float4*>(src);
                *reinterpret_cast<float4*>(dst + 4) = *reinterpret_cast<const float4*>(src + 4);
            }
        }
    } else {
        for (int k = 0; k < nt; ++k)
            for (int i = threadIdx.x; i < W; i += ROUTE_THREADS) rows[(size_t)k * W + i] = to_f32<TH>(h[(size_t)(t0 + k) * W + i]);
    }
    for (int k = nt; k < ROUTE_TOK; ++k)
        for (int i = threadIdx.x; i < W; i += ROUTE_THREADS) rows[(size_t)k * W + i] = 0.f;
    __syncthreads();
    // A warp takes up to RE outputs side by side (a row's elements are read once for them), a lane eight neighbouring
    // elements a load where the rows allow it (16-byte loads, several in flight), else one.  Either way the order of a dot
    // product's additions is fixed by W alone.  (Index E is the row beside the router's, when there is one.)
    constexpr int RE = ROUTE_TOK > 1 ? 3 : 1, RW = ROUTE_THREADS / 32, UNROLL = ROUTE_TOK > 1 ? 2 : 8;
    const bool wide = (W & 7) == 0 && (((size_t)w_router | (size_t)row_w) & 15) == 0;
    const int outputs = E + (row_w ? 1 : 0);
    for (int e0 = warp; e0 < outputs; e0 += RW * RE) {
        const TW* wr[RE];
        float acc[RE][ROUTE_TOK];
#pragma unroll
        for (int x = 0; x < RE; ++x) {
            const int e = min(e0 + x * RW, outputs - 1);
            wr[x] = e < E ? w_router + (size_t)e * W : row_w;
#pragma unroll
            for (int k = 0; k < ROUTE_TOK; ++k) acc[x][k] = 0.f;
        }
        if (wide) {
#pragma unroll UNROLL
            for (int i = lane * 8; i < W; i += 256) {
                float w8[RE][8];
#pragma unroll
                for (int x = 0; x < RE; ++x) {
                    if constexpr (sizeof(TW) == 2) {
                        const uint4 raw = *reinterpret_cast<const uint4*>(wr[x] + i);
                        const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
                        for (int k = 0; k < 4; ++k) { const float2 f = __bfloat1622float2(p2[k]); w8[x][2 * k] = f.x; w8[x][2 * k + 1] = f.y; }
                    } else {
                        const float4 a = *reinterpret_cast<const float4*>(wr[x] + i), b = *reinterpret_cast<const float4*>(wr[x] + i + 4);
                        w8[x][0] = a.x; w8[x][1] = a.y; w8[x][2] = a.z; w8[x][3] = a.w; w8[x][4] = b.x; w8[x][5] = b.y; w8[x][6] = b.z; w8[x][7] = b.w;
                    }
                }
#pragma unroll
                for (int k = 0; k < ROUTE_TOK; ++k) {
                    const float* row = rows + (size_t)k * W + i;
                    const float4 r0 = *reinterpret_cast<const float4*>(row), r1 = *reinterpret_cast<const float4*>(row + 4);
#pragma unroll
                    for (int x = 0; x < RE; ++x) {
                        float a = acc[x][k];
                        a = fmaf(r0.x, w8[x][0], a); a = fmaf(r0.y, w8[x][1], a); a = fmaf(r0.z, w8[x][2], a); a = fmaf(r0.w, w8[x][3], a);
                        a = fmaf(r1.x, w8[x][4], a); a = fmaf(r1.y, w8[x][5], a); a = fmaf(r1.z, w8[x][6], a); a = fmaf(r1.w, w8[x][7], a);
                        acc[x][k] = a;
                    }
                }
            }
        } else {
            for (int i = lane; i < W; i += 32) {
#pragma unroll
                for (int x = 0; x < RE; ++x) {
                    const float wv = to_f32<TW>(wr[x][i]);
#pragma unroll
                    for (int k = 0; k < ROUTE_TOK; ++k) acc[x][k] = fmaf(rows[(size_t)k * W + i], wv, acc[x][k]);
                }
            }
        }
#pragma unroll
        for (int x = 0; x < RE; ++x) {
            const int e = e0 + x * RW;
            if (e >= outputs) continue;
#pragma unroll
            for (int k = 0; k < ROUTE_TOK; ++k) {
                if (e == E) {
                    const float z = warp_sum(acc[x][k]);
                    if (lane == 0 && k < nt) row_out[t0 + k] = 1.0f / (1.0f + expf(-z));
                    continue;
                }
                const float z = warp_sum(acc[x][k]) + (bias ? bias[e] : 0.f);
                if (lane == 0) scores[(size_t)k * 3 * E + e] = softmax_scores ? z : 1.0f / (1.0f + expf(-z));
            }
        }
    }
    __syncthreads();
    if (warp >= nt) return;                    // warp i: token t0 + i
    const int t = t0 + warp;
    float* score = scores + (size_t)warp * 3 * E;
    float* choice = score + E;
    float* gbest = choice + E;
    if (softmax_scores == 1) {                 // over all router outputs, in an order that E alone fixes
        float m = -INFINITY;
        for (int e = lane; e < E; e += 32) m = fmaxf(m, score[e]);
        m = warp_max(m);
        float sum = 0.f;
        for (int e = lane; e < E; e += 32) { const float x = expf(score[e] - m); score[e] = x; sum += x; }
        sum = warp_sum(sum);
        __syncwarp();
        for (int e = lane; e < E; e += 32) score[e] = score[e] / sum;
        __syncwarp();
    }
    for (int e = lane; e < E; e += 32) choice[e] = score[e] + (correction ? correction[e] : 0.f);
    __syncwarp();
    if (groups > 1 && keep < groups) {         // only the experts of the ``keep`` groups with the best member stay
        const int per = E / groups;
        for (int g = lane; g < groups; g += 32) {
            float b = -INFINITY;
            for (int j = 0; j < per; ++j) b = fmaxf(b, choice[g * per + j]);
            gbest[g] = b;
        }
        __syncwarp();
        for (int k = 0; k < keep; ++k) {
            float best = -INFINITY; int arg = 0x7fffffff;
            for (int g = lane; g < groups; g += 32) {
                const float s = gbest[g];
                if (!isnan(s) && (arg == 0x7fffffff || s > best)) { best = s; arg = g; }   // kept groups are NaN
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ob = __shfl_xor_sync(0xffffffffu, best, o);
                const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
                if (oa != 0x7fffffff && (arg == 0x7fffffff || ob > best || (ob == best && oa < arg))) { best = ob; arg = oa; }
            }
            if (lane == 0 && arg != 0x7fffffff) gbest[arg] = __int_as_float(0x7fc00000);   // NaN marks a kept group
            __syncwarp();
        }
        for (int e = lane; e < E; e += 32)
            if (!isnan(gbest[e / per])) choice[e] = -INFINITY;
        __syncwarp();
    }
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY; int arg = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            const float s = choice[e];
            if (s > best) { best = s; arg = e; }      // ascending e: the first of equals stays
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
            if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
        }
        const float wgt = arg != 0x7fffffff ? score[arg] : 0.f;   // the weight is the score without the correction
        if (lane == 0) {
            // an identity expert (index >= num_real) has no rows among the experts' products: -1
            pair_expert[(size_t)t * top + k] = (arg == 0x7fffffff || arg >= num_real) ? -1 : arg;
            pair_weight[(size_t)t * top + k] = wgt;
            if (arg != 0x7fffffff) {
                if (arg < num_real) atomicAdd(&counts[arg], 1);
                choice[arg] = -INFINITY;              // taken
            }
        }
        total += wgt;
        __syncwarp();
    }
    if (softmax_scores == 2) {                 // the scores are the logits themselves: softmax over the chosen ones only
        if (lane == 0) {
            float* pw = pair_weight + (size_t)t * top;
            float m = -INFINITY, sum = 0.f;
            for (int k = 0; k < top; ++k) m = fmaxf(m, pw[k]);
            for (int k = 0; k < top; ++k) { pw[k] = expf(pw[k] - m); sum += pw[k]; }
            for (int k = 0; k < top; ++k) pw[k] /= sum;
        }
        return;
    }
    if (renormalize && lane == 0)
        for (int k = 0; k < top; ++k) pair_weight[(size_t)t * top + k] /= total + 1e-20f;   // (all chosen scores may be zero)
}

// pad_rows > 0: every expert's rows start at a multiple of pad_rows (= tile_rows): the sorted order then consists of
// whole tiles of one expert each, and lane_group[row / pad_rows] names it (-1: a tile nobody uses), which is what the
// grouped tcgen05 product reads.
// The first row and the first tile of every expert from the experts' counts, by one warp, 32 experts at a time.
__device__ __forceinline__ void layout_experts(const int* count, int E, int tile_rows, int pad_rows, int* first, int* tile0,
                                               int* num_tiles) {
    const int lane = threadIdx.x & 31;
    int rows = 0, tiles = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
        const int e = e0 + lane;
        const int c = e < E ? count[e] : 0;
        int r = pad_rows > 0 ? (c + pad_rows - 1) / pad_rows * pad_rows : c, n = (c + tile_rows - 1) / tile_rows;
        const int own_r = r, own_n = n;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int a = __shfl_up_sync(0xffffffffu, r, o), b = __shfl_up_sync(0xffffffffu, n, o);
            if (lane >= o) { r += a; n += b; }
        }
        if (e < E) { first[e] = rows + r - own_r; tile0[e] = tiles + n - own_n; }
        rows += __shfl_sync(0xffffffffu, r, 31);
        tiles += __shfl_sync(0xffffffffu, n, 31);
    }
    if (lane == 0) *num_tiles = tiles;
}

__global__ void __launch_bounds__(256)
moe_plan_kernel(int* __restrict__ counts, int E, int tile_rows, int* __restrict__ cursor,
                int* __restrict__ tile_group, int* __restrict__ tile_row0, int* __restrict__ tile_row_end,
                int* __restrict__ num_tiles, int pad_rows, int* __restrict__ lane_group, int lane_tiles) {
    extern __shared__ int smi[];
    int* count = smi;                          // [E]
    int* first = smi + E;                      // [E]
    int* tile0 = first + E;                    // [E]
    pdl_launch_dependents();
    pdl_wait();
    for (int e = threadIdx.x; e < E; e += 256) { count[e] = __ldcg(counts + e); counts[e] = 0; }
    if (lane_group)
        for (int i = threadIdx.x; i < lane_tiles; i += 256) lane_group[i] = -1;
    __syncthreads();
    if (threadIdx.x < 32) layout_experts(count, E, tile_rows, pad_rows, first, tile0, num_tiles);
    __syncthreads();
    for (int e = threadIdx.x; e < E; e += 256) {
        const int c = count[e], off = first[e];
        int n = tile0[e];
        cursor[e] = off;
        for (int r = off; r < off + c; r += tile_rows, ++n) {
            tile_group[n] = e; tile_row0[n] = r; tile_row_end[n] = off + c;
            if (lane_group) lane_group[r / pad_rows] = e;
        }
    }
}

constexpr int TABLE_THREADS = 1024;

__global__ void __launch_bounds__(TABLE_THREADS)
moe_table_kernel(const int* __restrict__ tokens, const int* __restrict__ table, int table_rows, int P, int top, int E,
                 int tile_rows, int pad_rows, int* __restrict__ pair_expert, float* __restrict__ pair_weight,
                 int* __restrict__ row_map, int* __restrict__ token_of_row, int* __restrict__ place_of_pair,
                 int* __restrict__ tile_group, int* __restrict__ tile_row0, int* __restrict__ tile_row_end,
                 int* __restrict__ num_tiles, int* __restrict__ lane_group, int lane_tiles, int* __restrict__ counts) {
    extern __shared__ int smi[];
    int* count = smi;                          // [E] pairs of the expert, later its cursor
    int* first = smi + E;                      // [E] its first row
    int* tile0 = first + E;                    // [E] its first tile
    pdl_launch_dependents();
    const int tid = threadIdx.x;
    for (int e = tid; e < E; e += TABLE_THREADS) count[e] = 0;
    __syncthreads();
    pdl_wait();
    if (lane_group)
        for (int i = tid; i < lane_tiles; i += TABLE_THREADS) lane_group[i] = -1;
    if (!table) {                              // the router's choice: count it; its counters go back to zero
        for (int e = tid; e < E; e += TABLE_THREADS) counts[e] = 0;
        for (int i = tid; i < P; i += TABLE_THREADS) {
            const int e = __ldcg(pair_expert + i);
            if (e >= 0) atomicAdd(&count[e], 1);
        }
    }
    const float w = 1.0f / (float)top;
    for (int i = tid; table && i < P; i += TABLE_THREADS) {
        const int tok = tokens[i / top];
        int e = (tok >= 0 && tok < table_rows) ? table[(size_t)tok * top + i % top] : -1;
        if (e < 0 || e >= E) e = -1;           // the host refuses such ids and tables; never a wrong row
        pair_expert[i] = e;
        pair_weight[i] = w;
        if (e >= 0) atomicAdd(&count[e], 1);
    }
    __syncthreads();
    if (tid < 32) layout_experts(count, E, tile_rows, pad_rows, first, tile0, num_tiles);
    __syncthreads();
    for (int e = tid; e < E; e += TABLE_THREADS) {
        const int c = count[e], r0 = first[e];
        int n = tile0[e];
        for (int r = r0; r < r0 + c; r += tile_rows, ++n) {
            tile_group[n] = e; tile_row0[n] = r; tile_row_end[n] = r0 + c;
            if (lane_group) lane_group[r / pad_rows] = e;
        }
        count[e] = r0;                         // from here on the cursor
    }
    __syncthreads();
    for (int i = tid; i < P; i += TABLE_THREADS) {
        const int e = table ? pair_expert[i] : __ldcg(pair_expert + i);        // (this thread wrote it, or the router's kernel)
        const int place = e >= 0 ? atomicAdd(&count[e], 1) : -1;
        if (place >= 0) { row_map[place] = i; token_of_row[place] = i / top; }
        if (place_of_pair) place_of_pair[i] = place;
    }
}

// x[place_of_pair[pair]] = h[pair / top]; rows of whole tiles beyond an expert's own are left as they are (their products
// are never read).
template <typename TH>
__global__ void __launch_bounds__(128)
moe_spread_kernel(const TH* __restrict__ h, int W, int top, const int* __restrict__ place_of_pair, TH* __restrict__ x) {
    pdl_launch_dependents();
    pdl_wait();
    const int place = __ldcg(place_of_pair + blockIdx.x);
    if (place < 0) return;
    const TH* src = h + (size_t)(blockIdx.x / top) * W;
    TH* dst = x + (size_t)place * W;
    constexpr int N = 16 / sizeof(TH);
    if (W % N == 0 && (((uintptr_t)h | (uintptr_t)x) & 15) == 0) {
        for (int i = threadIdx.x; i < W / N; i += 128)
            reinterpret_cast<uint4*>(dst)[i] = __ldcg(reinterpret_cast<const uint4*>(src) + i);
    } else {
        for (int i = threadIdx.x; i < W; i += 128) dst[i] = src[i];
    }
}

template <typename TH>
__global__ void __launch_bounds__(128)
moe_gather_kernel(const TH* __restrict__ h, int W, int top, const int* __restrict__ pair_expert,
                  const float* __restrict__ pair_weight, int weight_on_input, int* __restrict__ cursor,
                  int* __restrict__ row_map, int* __restrict__ place_of_pair, TH* __restrict__ x) {
    __shared__ int place_s;
    pdl_launch_dependents();
    pdl_wait();
    const int pair = blockIdx.x;
    const int expert = pair_expert[pair];
    if (expert < 0) {                                 // an identity expert: no row among the experts' products
        if (threadIdx.x == 0 && place_of_pair) place_of_pair[pair] = -1;
        return;
    }
    if (threadIdx.x == 0) {
        place_s = atomicAdd(&cursor[expert], 1);
        row_map[place_s] = pair;
        if (place_of_pair) place_of_pair[pair] = place_s;
    }
    __syncthreads();
    const int place = place_s;
    const float w = weight_on_input ? pair_weight[pair] : 1.f;
    const TH* src = h + (size_t)(pair / top) * W;
    TH* dst = x + (size_t)place * W;
    for (int i = threadIdx.x; i < W; i += 128) dst[i] = from_f32<TH>(w * to_f32<TH>(src[i]));
}

// four neighbouring elements as float32
__device__ __forceinline__ float4 load_row4(const float* p) { return __ldcg(reinterpret_cast<const float4*>(p)); }
__device__ __forceinline__ float4 load_row4(const bf16* p) {
    const uint2 raw = __ldcg(reinterpret_cast<const uint2*>(p));
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

// VEC columns a thread (4: 16-byte accesses); pairs are asked for eight at a time
template <typename TH, int VEC>
__global__ void __launch_bounds__(256)
moe_combine_kernel(const float* __restrict__ y, int W, int top, const float* __restrict__ pair_weight,
                   int weight_on_output, const int* __restrict__ place_of_pair, float* __restrict__ residual,
                   float* __restrict__ out, const int* __restrict__ pair_expert, const TH* __restrict__ h,
                   float* __restrict__ shared, const float* __restrict__ shared_w, int clear_shared) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int i = (blockIdx.y * 256 + threadIdx.x) * VEC;
    if (i >= W) return;
    auto load = [&](const auto* p, float (&v)[VEC]) {
        if constexpr (VEC == 4) { const float4 x = load_row4(p); v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; }
        else v[0] = to_f32(*p);
    };
    float acc[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) acc[c] = 0.f;
    const size_t at = (size_t)t * W + i;
    for (int k0 = 0; k0 < top; k0 += 4) {
        float v[4][VEC], w[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            if (k0 + u >= top) continue;
            const size_t pair = (size_t)t * top + k0 + u;     // y in (token, rank) order, or in the sorted order
            if (pair_expert && __ldcg(pair_expert + pair) < 0) {       // an identity expert: the weight times the input itself
                w[u] = __ldcg(pair_weight + pair);
                load(h + at, v[u]);
                continue;
            }
            w[u] = weight_on_output ? __ldcg(pair_weight + pair) : 1.f;
            load(y + (place_of_pair ? (size_t)__ldcg(place_of_pair + pair) : pair) * W + i, v[u]);
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (k0 + u < top)
#pragma unroll
                for (int c = 0; c < VEC; ++c) acc[c] = fmaf(w[u], v[u][c], acc[c]);
    }
    if (shared) {                                             // an expert that every token uses, times the token's weight
        float v[VEC];
        load(shared + at, v);
        const float w = __ldcg(shared_w + t);
#pragma unroll
        for (int c = 0; c < VEC; ++c) acc[c] = fmaf(w, v[c], acc[c]);
        if (clear_shared)
#pragma unroll
            for (int c = 0; c < VEC; ++c) shared[at + c] = 0.f;
    }
    if (residual) {
        float v[VEC];
        load(residual + at, v);
#pragma unroll
        for (int c = 0; c < VEC; ++c) acc[c] += v[c];
    }
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(out + at) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    else out[at] = acc[0];
}

}  // namespace

// E router outputs, of which the last E - num_real are identity experts (pair_expert -1).  softmax_scores: the scores are
// softmax(z) over all E outputs instead of sigmoid(z); 2: the scores are the logits z, and the weights of the chosen are the
// softmax over the chosen logits alone.  bias [E] float32 or null: added to the router's product.  correction [E] float32 or null: added to the scores for the
// choice only.  row_w [W] (the router's type) or null: one more row, row_out[t] = sigmoid(row_w . h[t]).  groups > 1 with keep < groups: E / groups neighbours form a group, and only the ``keep`` groups whose best
// choice score is largest can be chosen from.
TFF_API int tff_moe_route(const void* h, int h_dt, const void* w_router, int w_dt, const float* bias, int T, int W, int E, int top,
                          int renormalize, int softmax_scores, const float* correction, int groups, int keep,
                          int num_real, int* pair_expert, float* pair_weight, int* counts, const void* row_w, float* row_out,
                          cudaStream_t stream) {
    if (T <= 0) return TFF_OK;
    if (W <= 0 || E <= 0 || top <= 0 || top > E || !h || !w_router || num_real < 0 || num_real > E || (row_w && !row_out))
        return TFF_ERR_BAD_ARGUMENT;
    if (groups > 1 && (E % groups != 0 || keep <= 0 || keep > groups || top > keep * (E / groups))) return TFF_ERR_BAD_ARGUMENT;
    const bool few = T <= ROUTE_FEW;
    const int tok = few ? ROUTE_FEW_TOK : ROUTE_MANY_TOK;
    const size_t smem = (size_t)tok * (W + 3 * E) * sizeof(float);
    if (smem > 200 * 1024) return TFF_ERR_UNSUPPORTED;
#define TFF_ROUTE_N(TH, TW, TOK, THREADS)                                                                             \
    do {                                                                                                              \
        if (smem > 48 * 1024)                                                                                         \
            cudaFuncSetAttribute(moe_route_kernel<TH, TW, TOK, THREADS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        return tff_launch_pdl(moe_route_kernel<TH, TW, TOK, THREADS>, dim3((T + TOK - 1) / TOK), dim3(THREADS), smem, stream, (const TH*)h, \
                              (const TW*)w_router, bias, T, W, E, top, renormalize, softmax_scores, correction, groups, keep, \
                              num_real, pair_expert, pair_weight, counts, (const TW*)row_w, row_out);         \
    } while (0)
#define TFF_ROUTE(TH, TW)                                                                                             \
    do {                                                                                                              \
        if (few) TFF_ROUTE_N(TH, TW, ROUTE_FEW_TOK, ROUTE_FEW_THREADS);                                               \
        TFF_ROUTE_N(TH, TW, ROUTE_MANY_TOK, ROUTE_MANY_THREADS);                                                      \
    } while (0)
    if (h_dt == 0 && w_dt == 0) TFF_ROUTE(float, float);
    if (h_dt == 0 && w_dt == 1) TFF_ROUTE(float, bf16);
    if (h_dt == 1 && w_dt == 1) TFF_ROUTE(bf16, bf16);
    if (h_dt == 1 && w_dt == 0) TFF_ROUTE(bf16, float);
#undef TFF_ROUTE
#undef TFF_ROUTE_N
    return TFF_ERR_BAD_ARGUMENT;
}

TFF_API int tff_moe_plan(int* counts, int E, int tile_rows, int* cursor, int* tile_group, int* tile_row0,
                         int* tile_row_end, int* num_tiles, int pad_rows, int* lane_group, int lane_tiles,
                         cudaStream_t stream) {
    if (E <= 0 || tile_rows <= 0 || pad_rows < 0 || (pad_rows > 0 && pad_rows != tile_rows) || (lane_group && pad_rows <= 0))
        return TFF_ERR_BAD_ARGUMENT;
    if (E > 4096) return TFF_ERR_UNSUPPORTED;
    return tff_launch_pdl(moe_plan_kernel, dim3(1), dim3(256), (size_t)3 * E * sizeof(int), stream, counts, E, tile_rows, cursor, tile_group,
                          tile_row0, tile_row_end, num_tiles, pad_rows, lane_group, lane_tiles);
}

// tokens [P / top] int32, table [table_rows, top] int32.  Outputs as tff_moe_route, tff_moe_plan and tff_moe_gather leave
// them (place_of_pair and lane_group may be null), and token_of_row: sorted place -> row of the step's tokens.  With table null
// pair_expert is the choice that tff_moe_route left, and its ``counts`` are set back to zero.
TFF_API int tff_moe_table(const int* tokens, const int* table, int table_rows, int P, int top, int E, int tile_rows,
                          int pad_rows, int* pair_expert, float* pair_weight, int* row_map, int* token_of_row,
                          int* place_of_pair, int* tile_group, int* tile_row0, int* tile_row_end, int* num_tiles,
                          int* lane_group, int lane_tiles, int* counts, cudaStream_t stream) {
    if (P <= 0) return TFF_OK;
    if ((table ? !tokens || table_rows <= 0 : !counts) || top <= 0 || P % top || E <= 0 || tile_rows <= 0 || pad_rows < 0 ||
        (pad_rows > 0 && pad_rows != tile_rows) || (lane_group && pad_rows <= 0) || !pair_expert || !pair_weight || !row_map ||
        !token_of_row || !tile_group || !tile_row0 || !tile_row_end || !num_tiles)
        return TFF_ERR_BAD_ARGUMENT;
    const size_t smem = (size_t)3 * E * sizeof(int);
    if (smem > 48 * 1024) return TFF_ERR_UNSUPPORTED;
    return tff_launch_pdl(moe_table_kernel, dim3(1), dim3(TABLE_THREADS), smem, stream, tokens, table, table_rows, P, top, E,
                          tile_rows, pad_rows, pair_expert, pair_weight, row_map, token_of_row, place_of_pair, tile_group,
                          tile_row0, tile_row_end, num_tiles, lane_group, lane_tiles, counts);
}

TFF_API int tff_moe_spread(const void* h, int h_dt, int pairs, int W, int top, const int* place_of_pair, void* x,
                           cudaStream_t stream) {
    if (pairs <= 0) return TFF_OK;
    if (!h || !x || !place_of_pair || top <= 0 || W <= 0) return TFF_ERR_BAD_ARGUMENT;
    if (h_dt == 0)
        return tff_launch_pdl(moe_spread_kernel<float>, dim3(pairs), dim3(128), 0, stream, (const float*)h, W, top, place_of_pair, (float*)x);
    return tff_launch_pdl(moe_spread_kernel<bf16>, dim3(pairs), dim3(128), 0, stream, (const bf16*)h, W, top, place_of_pair, (bf16*)x);
}

TFF_API int tff_moe_gather(const void* h, int h_dt, int pairs, int W, int top, const int* pair_expert,
                           const float* pair_weight, int weight_on_input, int* cursor, int* row_map,
                           int* place_of_pair, void* x, cudaStream_t stream) {
    if (pairs <= 0) return TFF_OK;
    if (h_dt == 0)
        return tff_launch_pdl(moe_gather_kernel<float>, dim3(pairs), dim3(128), 0, stream, (const float*)h, W, top,
                              pair_expert, pair_weight, weight_on_input, cursor, row_map, place_of_pair, (float*)x);
    return tff_launch_pdl(moe_gather_kernel<bf16>, dim3(pairs), dim3(128), 0, stream, (const bf16*)h, W, top,
                          pair_expert, pair_weight, weight_on_input, cursor, row_map, place_of_pair, (bf16*)x);
}

// pair_expert (null: every pair has a row in y) and h [T, W] (h_dt 0 float32, 1 bfloat16): pairs whose expert is -1 are
// identity experts and add pair_weight * h[t]; pair_weight must then be given.  shared [T, W] and shared_w [T] (or null): the
// rows of an expert that every token uses and their weights; clear_shared: the rows are set to zero behind the read.
TFF_API int tff_moe_combine(const float* y, int T, int W, int top, const float* pair_weight, int weight_on_output,
                            const int* place_of_pair, float* residual, float* out, const int* pair_expert,
                            const void* h, int h_dt, float* shared, const float* shared_w, int clear_shared,
                            cudaStream_t stream) {
    if (T <= 0) return TFF_OK;
    if (shared && !shared_w) return TFF_ERR_BAD_ARGUMENT;
    if (pair_expert && (!h || !pair_weight)) return TFF_ERR_BAD_ARGUMENT;
    const bool vec = W % 4 == 0 && (((uintptr_t)y | (uintptr_t)residual | (uintptr_t)out | (uintptr_t)h | (uintptr_t)shared) & 15) == 0;
    const int cols = vec ? W / 4 : W;
    const dim3 grid(T, (cols + 255) / 256), block(cols < 256 ? (cols + 31) / 32 * 32 : 256);
#define TFF_COMBINE(TH, VEC)                                                                                          \
    return tff_launch_pdl(moe_combine_kernel<TH, VEC>, grid, block, 0, stream, y, W, top, pair_weight, weight_on_output, \
                          place_of_pair, residual, out, pair_expert, (const TH*)h, shared, shared_w, clear_shared)
    if (h_dt == 1) { if (vec) TFF_COMBINE(bf16, 4); TFF_COMBINE(bf16, 1); }
    if (vec) TFF_COMBINE(float, 4);
    TFF_COMBINE(float, 1);
#undef TFF_COMBINE
}

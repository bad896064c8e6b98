// The matrix memory of xLSTM (mLSTM): linear attention over a matrix state per head whose input and forget gates are
// exponentials read from the token, held in range by a running maximum, with a normaliser that follows the keys.
//   i_t = cap tanh((zi_t + bi) / cap),  f_t = logsigmoid(cap tanh((zf_t + bf) / cap))          one of each per head and token
//   m_t = max(f_t + m_(t-1), i_t)                                                             m = 0 ahead of the first token
//   S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T      S [d, dv] per (request, head), zeros at the start
//   n_t = e^(f_t + m_(t-1) - m_t) n_(t-1) + e^(i_t - m_t) k_t            n [d]
//   o_t = S_t^T q_t / (max(|n_t . q_t|, e^-m_t) + 1e-6)                   q_t the projection times q_scale
// q, k, v and the gates' inputs zi, zf are column blocks of float32 rows (a mixer's merged projection); o goes to float32 rows
// [T, H*dv].  state [slots, slot_len]: a slot holds S of all heads [H, d, dv], then n [H, d], then m [H].  A request that
// brings position 0 starts from zeros whatever its slot holds.
//
// Token by token (steps of one token a request; everything in the 32-bit mode): a CTA per (head, request); the state streams
// through registers, and stays there over the tokens of a portion where it fits.  All float32 FMAs.
//
// Chunk by chunk on the tensor cores (chunk_recurrence.cuh; portions of prompts).  With F_t the sum of the f from the chunk's
// first token to t, a_s = i_s - F_s and M_t = max over s <= t of a_s, a chunk that starts from (S_0, n_0, m_0) has
//   m_t = F_t + M'_t,   M'_t = max(m_0, M_t)
//   S_t^T q_t = sum_(s<=t) e^(a_s - M'_t) (q_t . k_s) v_s + e^(m_0 - M'_t) S_0^T q_t,   n_t . q_t likewise without v
// The local kernel (a CTA per chunk and head, all chunks at once) computes the sums with M_t in place of M'_t, which needs
// nothing of earlier chunks; the scan walks the chunks with S, n and m; the finish kernel (a CTA per chunk, head and block of
// value columns) puts e^(M_t - M'_t) on the local part, adds the start state's and divides.
// The exponents never exceed zero, so nothing overflows.
#include "chunk_recurrence.cuh"
#include <type_traits>

namespace {

struct MlstmParams {
    const float* proj; int ld, q_off, k_off, v_off, i_off, f_off;
    const float* gate_bias;            // [2 H]: the input gates' biases, then the forget gates'
    float cap, q_scale;
    float* state; int num_slots, slot_len;
    const int* q_start; const int* pos_start; const int* slots;
    float* out; int H, d, dv;
    // The step kernel may go on to the mixer's output: mixed[t, h*dv + j] = o_j / rms(o) * norm_w[h*dv + j] * sigmoid(g), g the
    // row's columns g_off .. (norm_w null: o itself to ``out``); with ``clear`` it sets what it has read of the row to zero.
    float* rows; int g_off; const float* norm_w; float eps; void* mixed; int mixed_is_bf16, clear;
};

__device__ __forceinline__ float in_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float forget_gate(float z, float cap) {      // log of a sigmoid
    const float x = cap * tanhf(z / cap);
    return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}
__device__ __forceinline__ float divide(float num, float nq, float m) { return num / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f); }

// ------------------------------------------------------------------ token by token
// Threads of a CTA: small ones, four an SM, for steps of one token of many requests, which stream the states (64 requests of 16
// heads of 128 x 128: 35 us against 43, 57 with one large CTA an SM); large ones, whose registers hold such a head, for few
// requests and for portions.  ROWS: rows of a column group that a thread has in flight.
constexpr int FEW = 256, MANY = 512, ROWS = 8;

// VEC value columns a thread; KEEP: the head's state stays in registers (ROWS rows a thread and one column group cover it)
template <int VEC, bool KEEP, int ST>
__global__ void __launch_bounds__(ST, ST == FEW ? 4 : 2)
mlstm_step_kernel(MlstmParams p) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[32];
    typedef typename std::conditional<VEC == 4, float4, float>::type V;
    pdl_launch_dependents();
    const int h = blockIdx.x, b = blockIdx.y, d = p.d, dv = p.dv, tid = threadIdx.x;
    float* sq = sm;                     // [d]
    float* sk = sq + d;                 // [d]
    float* sn = sk + d;                 // [d]
    float* so = sn + d;                 // [dv]
    float* part = so + dv;              // [NY][groups * VEC]
    const int groups = (dv + VEC - 1) / VEC, LX = min(groups, ST), NY = ST / LX;
    const int lx = tid % LX, ty = tid / LX;
    const int t0 = p.q_start[b], t1 = p.q_start[b + 1];
    const int slot = p.slots[b];
    const bool ok = t1 > t0 && slot >= 0 && slot < p.num_slots;
    float* base = p.state + (size_t)(ok ? slot : 0) * p.slot_len;
    float* S = base + (size_t)h * d * dv;
    float* N = base + (size_t)p.H * d * dv + (size_t)h * d;
    float* Mx = base + (size_t)p.H * d * dv + (size_t)p.H * d + h;
    bool fresh = p.pos_start[b] == 0;
    if (ok && !fresh)                   // into the second-level cache while the kernels ahead are still at work
        for (int e = tid * 32; e < d * dv; e += ST * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(S + e));
    pdl_wait();
    if (!ok) return;
    V s[ROWS];
    auto load_rows = [&](int i0, int g) {
#pragma unroll
        for (int u = 0; u < ROWS; ++u) {
            const int i = i0 + u * NY;
            if constexpr (VEC == 4) s[u] = make_float4(0.f, 0.f, 0.f, 0.f); else s[u] = 0.f;
            if (ty < NY && i < d && !fresh) s[u] = __ldcg(reinterpret_cast<const V*>(S + (size_t)i * dv + g * VEC));
        }
    };
    if (KEEP) load_rows(ty, lx);
    for (int i = tid; i < d; i += ST) sn[i] = fresh ? 0.f : __ldcg(N + i);
    float m = fresh ? 0.f : __ldcg(Mx);
    for (int t = t0; t < t1; ++t) {
        const float* row = p.proj + (size_t)t * p.ld;
        __syncthreads();
        for (int i = tid; i < d; i += ST) {
            sq[i] = __ldcg(row + p.q_off + h * d + i) * p.q_scale;
            sk[i] = __ldcg(row + p.k_off + h * d + i);
        }
        const float ig = in_gate(__ldcg(row + p.i_off + h) + p.gate_bias[h], p.cap);
        const float fg = forget_gate(__ldcg(row + p.f_off + h) + p.gate_bias[p.H + h], p.cap);
        const float m_new = fmaxf(fg + m, ig);
        const float keep = expf(fg + m - m_new), take = expf(ig - m_new);
        m = m_new;
        __syncthreads();
        float nq = 0.f;
        for (int i = tid; i < d; i += ST) {              // (this thread alone reads and writes its elements of n)
            const float x = fmaf(keep, sn[i], take * sk[i]);
            sn[i] = x;
            nq = fmaf(x, sq[i], nq);
        }
        for (int g = lx; g < groups && ty < NY; g += LX) {
            float v[VEC], acc[VEC];
#pragma unroll
            for (int c = 0; c < VEC; ++c) {
                v[c] = take * __ldcg(row + p.v_off + (size_t)h * dv + g * VEC + c);
                acc[c] = 0.f;
            }
            for (int i0 = ty; i0 < d; i0 += NY * ROWS) {
                if (!KEEP) load_rows(i0, g);
#pragma unroll
                for (int u = 0; u < ROWS; ++u) {
                    const int i = i0 + u * NY;
                    if (i >= d) continue;
                    const float ki = sk[i], qi = sq[i];
                    float* e = reinterpret_cast<float*>(&s[u]);
#pragma unroll
                    for (int c = 0; c < VEC; ++c) {
                        e[c] = fmaf(keep, e[c], ki * v[c]);
                        acc[c] = fmaf(e[c], qi, acc[c]);
                    }
                    if (!KEEP) *reinterpret_cast<V*>(S + (size_t)i * dv + g * VEC) = s[u];
                }
            }
#pragma unroll
            for (int c = 0; c < VEC; ++c) part[(size_t)ty * groups * VEC + g * VEC + c] = acc[c];
        }
        nq = block_sum<ST>(nq, red);                     // (a barrier behind the partial sums too)
        float ss = 0.f;
        for (int j = tid; j < dv; j += ST) {
            float o = 0.f;
            for (int y = 0; y < NY; ++y) o += part[(size_t)y * groups * VEC + j];
            o = divide(o, nq, m);
            if (!p.norm_w) { p.out[(size_t)t * p.H * dv + (size_t)h * dv + j] = o; continue; }
            so[j] = o;                                   // (this thread alone reads it back)
            ss = fmaf(o, o, ss);
        }
        fresh = false;
        if (!p.norm_w) continue;
        const float inv = rsqrtf(block_sum<ST>(ss, red) / (float)dv + p.eps);
        float* wrow = p.rows + (size_t)t * p.ld;
        for (int j = tid; j < dv; j += ST) {
            const int c = h * dv + j;
            const float g = __ldcg(row + p.g_off + c);
            const float y = (so[j] * inv) * p.norm_w[c] / (1.0f + expf(-g));
            const size_t at = (size_t)t * p.H * dv + c;
            if (p.mixed_is_bf16) ((bf16*)p.mixed)[at] = __float2bfloat16_rn(y);
            else ((float*)p.mixed)[at] = y;
            if (p.clear) { wrow[p.g_off + c] = 0.f; wrow[p.v_off + c] = 0.f; }
        }
        if (p.clear) {                                   // (everything of the row that this head reads has been read)
            for (int i = tid; i < d; i += ST) { wrow[p.q_off + h * d + i] = 0.f; wrow[p.k_off + h * d + i] = 0.f; }
            if (tid == 0) { wrow[p.i_off + h] = 0.f; wrow[p.f_off + h] = 0.f; }
        }
    }
    if (KEEP && ty < NY && lx < groups)
#pragma unroll
        for (int u = 0; u < ROWS; ++u) {
            const int i = ty + u * NY;
            if (i < d) *reinterpret_cast<V*>(S + (size_t)i * dv + lx * VEC) = s[u];
        }
    for (int i = tid; i < d; i += ST) N[i] = sn[i];
    if (tid == 0) *Mx = m;
}

// ------------------------------------------------------------------ chunk by chunk
// Workspace: per (chunk, head) the end state of the chunk alone, which the scan replaces by the state the chunk starts from
// [S d*dv | n d], and numbers of its tokens.
__host__ __device__ inline int round4(int x) { return (x + 3) & ~3; }
__host__ __device__ inline int chunk_floats(int d, int dv) { return round4(d * dv) + round4(d); }
constexpr int NUMS = 3 * C + 4;        // M [C], F [C], the local n . q [C], the m the chunk starts from

struct Workspace { float* U; float* nums; };
__host__ __device__ inline Workspace workspace_of(float* ws, long long chunks, int H, int d, int dv) {
    return Workspace{ws, ws + chunks * H * chunk_floats(d, dv)};
}

struct LocalWeights {
    static constexpr bool SUMS = true;
    const float* a; const float* M; const float* tails;
    float scale;
    float* sums;
    __device__ __forceinline__ float pair(int i, int j) const { return scale * expf(a[j] - M[i]); }
    __device__ __forceinline__ float tail(int j) const { return tails[j]; }
    __device__ __forceinline__ void row_sum(int i, float x) const { sums[i] = x; }
};

__global__ void __launch_bounds__(MT, 2)
mlstm_local_kernel(MlstmParams p, int num_requests, Workspace w) {
    extern __shared__ __align__(16) unsigned char smraw[];
    __shared__ float sa[C], sM[C], tails[C];
    pdl_launch_dependents();
    const int h = blockIdx.y, d = p.d, dv = p.dv, lane = threadIdx.x & 31;
    ChunkRef c;
    const bool have = find_chunk(p.q_start, p.pos_start, num_requests, blockIdx.x, c);
    pdl_wait();
    if (!have) return;
    const size_t at = (size_t)blockIdx.x * p.H + h;
    float* nums = w.nums + at * NUMS;
    if (threadIdx.x < 32) {             // the chunk's gates: two tokens a lane, sums and maxima across the warp
        float fs[2], ig[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int j = 2 * lane + u;
            const float* row = p.proj + (size_t)(c.t + min(j, c.n - 1)) * p.ld;
            ig[u] = in_gate(__ldcg(row + p.i_off + h) + p.gate_bias[h], p.cap);
            fs[u] = j < c.n ? forget_gate(__ldcg(row + p.f_off + h) + p.gate_bias[p.H + h], p.cap) : 0.f;
        }
        float sum = fs[0] + fs[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += x;
        }
        float before = __shfl_up_sync(0xffffffffu, sum, 1);
        if (lane == 0) before = 0.f;
        const float F0 = before + fs[0], F1 = F0 + fs[1];
        const float a0 = ig[0] - F0, a1 = ig[1] - F1;
        const bool in0 = 2 * lane < c.n, in1 = 2 * lane + 1 < c.n;
        float top = fmaxf(in0 ? a0 : -INFINITY, in1 ? a1 : -INFINITY);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(0xffffffffu, top, o);
            if (lane >= o) top = fmaxf(top, x);
        }
        float ahead = __shfl_up_sync(0xffffffffu, top, 1);
        if (lane == 0) ahead = -INFINITY;
        const float M0 = in0 ? fmaxf(ahead, a0) : top, M1 = top;       // (tokens beyond the last: the chunk's maximum)
        sa[2 * lane] = in0 ? a0 : M0; sa[2 * lane + 1] = in1 ? a1 : M1;
        sM[2 * lane] = M0; sM[2 * lane + 1] = M1;
        nums[2 * lane] = M0; nums[2 * lane + 1] = M1;
        nums[C + 2 * lane] = F0; nums[C + 2 * lane + 1] = F1;
        // the request's first chunk of the step starts from the slot's m; the scan fills in the other chunks'
        if (lane == 0 && c.t == p.q_start[c.b]) {
            const int slot = p.slots[c.b];
            float m = 0.f;
            if (c.pos > 0 && slot >= 0 && slot < p.num_slots)
                m = __ldcg(p.state + (size_t)slot * p.slot_len + (size_t)p.H * d * dv + (size_t)p.H * d + h);
            nums[3 * C] = m;
        }
    }
    __syncthreads();
    const float* row = p.proj + (size_t)c.t * p.ld;
    float* Uc = w.U + at * chunk_floats(d, dv);
    const LocalWeights weights{sa, sM, tails, p.q_scale, nums + 2 * C};
    if (threadIdx.x < C) tails[threadIdx.x] = threadIdx.x < c.n ? expf(sa[threadIdx.x] - sM[c.n - 1]) : 0.f;
    chunk_local_mma(smraw, row + p.q_off + (size_t)h * d, p.ld, row + p.k_off + (size_t)h * d, p.ld, row + p.v_off + (size_t)h * dv,
                    p.ld, 0, c.n, d, dv, weights, p.out + (size_t)c.t * p.H * dv + (size_t)h * dv, p.H * dv, Uc);
    const bf16* Ks = local_keys(smraw, d);
    const int ks = pad16(d) + 8;
    for (int r = threadIdx.x; r < d; r += MT) {          // the normaliser's part: the keys' weighted sum
        float x = 0.f;
#pragma unroll 8
        for (int j = 0; j < C; ++j) x = fmaf(tails[j], __bfloat162float(Ks[j * ks + r]), x);
        Uc[round4(d * dv) + r] = x;
    }
}

// Per (request, head, element of S and n): the chunks in order.
template <int VEC>
__global__ void __launch_bounds__(256)
mlstm_scan_kernel(MlstmParams p, int num_requests, Workspace w) {
    pdl_launch_dependents();
    const int h = blockIdx.y, b = blockIdx.z, d = p.d, dv = p.dv;
    const int e = (blockIdx.x * 256 + threadIdx.x) * VEC;
    const int t0 = p.q_start[b], len = p.q_start[b + 1] - t0;
    const int slot = p.slots[b];
    int first_chunk = 0;                                               // chunks of the requests ahead of b
    for (int r = 0; r < b; ++r) {
        const int l = p.q_start[r + 1] - p.q_start[r];
        if (l > 0) first_chunk += (p.pos_start[r] + l - 1) / C - p.pos_start[r] / C + 1;
    }
    pdl_wait();
    if (len <= 0 || slot < 0 || slot >= p.num_slots || e >= d * dv + d) return;
    const int pos0 = p.pos_start[b];
    const int count = (pos0 + len - 1) / C - pos0 / C + 1;
    typedef typename std::conditional<VEC == 4, float4, float>::type V;
    float* base = p.state + (size_t)slot * p.slot_len;
    const bool is_n = e >= d * dv;
    V* gs = reinterpret_cast<V*>(is_n ? base + (size_t)p.H * d * dv + (size_t)h * d + (e - d * dv) : base + (size_t)h * d * dv + e);
    const int eu = is_n ? round4(d * dv) + e - d * dv : e;
    V S;
    if (pos0 == 0) { if constexpr (VEC == 4) S = make_float4(0.f, 0.f, 0.f, 0.f); else S = 0.f; }
    else S = __ldcg(gs);
    const size_t stride = (size_t)p.H * chunk_floats(d, dv);           // floats between a chunk's U and the next one's
    float* u0 = w.U + ((size_t)first_chunk * p.H + h) * chunk_floats(d, dv) + eu;
    float* nums = w.nums + ((size_t)first_chunk * p.H + h) * NUMS;
    float m = __ldcg(nums + 3 * C);
    for (int c0 = 0; c0 < count; c0 += 8) {                            // eight chunks are asked for together
        V add[8];
        float M[8], F[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int c = c0 + j;
            if (c >= count) continue;
            add[j] = __ldcg(reinterpret_cast<const V*>(u0 + (size_t)c * stride));
            const int lo = max(pos0, (pos0 / C + c) * C), hi = min(pos0 + len, (pos0 / C + c + 1) * C);
            const float* nc = nums + (size_t)c * p.H * NUMS + (hi - lo - 1);
            M[j] = __ldcg(nc);
            F[j] = __ldcg(nc + C);
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int c = c0 + j;
            if (c >= count) continue;
            if (e == 0 && c > 0) nums[(size_t)c * p.H * NUMS + 3 * C] = m;
            *reinterpret_cast<V*>(u0 + (size_t)c * stride) = S;
            const float top = fmaxf(m, M[j]), old = expf(m - top), take = expf(M[j] - top);
            m = F[j] + top;
            float* s = reinterpret_cast<float*>(&S);
            const float* a = reinterpret_cast<const float*>(&add[j]);
#pragma unroll
            for (int x = 0; x < VEC; ++x) s[x] = fmaf(old, s[x], take * a[x]);
        }
    }
    *gs = S;
    if (e == 0) base[(size_t)p.H * d * dv + (size_t)p.H * d + h] = m;
}

struct FinishWeights {
    const float* local; const float* start; const float* inv;
    __device__ __forceinline__ float join(int i, float dot, float part) const {
        return fmaf(start[i], dot, local[i] * part) * inv[i];
    }
};

__global__ void __launch_bounds__(MT, 2)
mlstm_finish_kernel(MlstmParams p, int num_requests, Workspace w) {
    extern __shared__ __align__(16) unsigned char smraw[];
    __shared__ float wl[C], ws[C], inv[C];
    pdl_launch_dependents();
    const int h = blockIdx.y, d = p.d, dv = p.dv, n0 = blockIdx.z * SCOLS;
    ChunkRef c;
    const bool have = find_chunk(p.q_start, p.pos_start, num_requests, blockIdx.x, c);
    pdl_wait();
    if (!have) return;
    const size_t at = (size_t)blockIdx.x * p.H + h;
    const float* Sc = w.U + at * chunk_floats(d, dv);
    const float* Nc = Sc + round4(d * dv);
    float* orow = p.out + (size_t)c.t * p.H * dv + (size_t)h * dv;
    FinishRegs f;
    chunk_finish_load(f, smraw, p.proj + (size_t)c.t * p.ld + p.q_off + (size_t)h * d, p.ld, 0, c.n, d, dv, n0, Sc, orow, p.H * dv);
    {   // the denominators: four threads a token
        const bf16* q = (const bf16*)smraw + (threadIdx.x >> 2) * (pad16(d) + 8);
        const int i = threadIdx.x >> 2;
        float nq = 0.f;
#pragma unroll 4
        for (int r = threadIdx.x & 3; r < d; r += 4) nq = fmaf(__bfloat162float(q[r]), __ldcg(Nc + r), nq);
        nq += __shfl_xor_sync(0xffffffffu, nq, 1);
        nq += __shfl_xor_sync(0xffffffffu, nq, 2);
        if ((threadIdx.x & 3) == 0 && i < c.n) {
            const float* nums = w.nums + at * NUMS;
            const float M = __ldcg(nums + i), F = __ldcg(nums + C + i), m0 = __ldcg(nums + 3 * C);
            const float top = fmaxf(m0, M), a = expf(M - top), s = expf(m0 - top) * p.q_scale;
            wl[i] = a; ws[i] = s;
            inv[i] = divide(1.f, fmaf(s, nq, a * __ldcg(nums + 2 * C + i)), F + top);
        }
    }
    __syncthreads();
    chunk_finish_mma(f, smraw, c.n, d, dv, n0, Sc, FinishWeights{wl, ws, inv}, orow, p.H * dv);
}

constexpr size_t MOST = 224 * 1024;    // dynamic shared memory a CTA may ask for here (the kernels have a little static on top)

int launch_chunked(const MlstmParams& p, int num_requests, float* workspace, int num_tokens, cudaStream_t stream) {
    if (!workspace || num_tokens <= 0) return TFF_ERR_BAD_ARGUMENT;
    const size_t smem1 = local_mma_smem(p.d, p.dv), smem3 = finish_mma_smem(p.d);
    if (smem1 > MOST || smem3 > MOST) return TFF_ERR_UNSUPPORTED;
    const int chunks = num_tokens / C + 2 * num_requests;
    const Workspace w = workspace_of(workspace, chunks, p.H, p.d, p.dv);
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(mlstm_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MOST) != cudaSuccess ||
            cudaFuncSetAttribute(mlstm_finish_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MOST) != cudaSuccess)
            return TFF_ERR_LAUNCH;
        configured = true;
    }
    int st = tff_launch_pdl(mlstm_local_kernel, dim3(chunks, p.H), dim3(MT), smem1, stream, p, num_requests, w);
    if (st != TFF_OK) return st;
    const int elements = p.d * p.dv + p.d;
    if (p.d % 4 == 0 && (((uintptr_t)p.state | (uintptr_t)workspace) & 15) == 0)      // (a slot's length is a multiple of 4)
        st = tff_launch_pdl(mlstm_scan_kernel<4>, dim3((elements / 4 + 255) / 256, p.H, num_requests), dim3(256), (size_t)0, stream,
                            p, num_requests, w);
    else
        st = tff_launch_pdl(mlstm_scan_kernel<1>, dim3((elements + 255) / 256, p.H, num_requests), dim3(256), (size_t)0, stream,
                            p, num_requests, w);
    if (st != TFF_OK) return st;
    return tff_launch_pdl(mlstm_finish_kernel, dim3(chunks, p.H, (p.dv + SCOLS - 1) / SCOLS), dim3(MT), smem3, stream, p,
                          num_requests, w);
}

}  // namespace

// Floats of workspace the chunked form needs for a step of ``num_tokens`` tokens in ``num_requests`` requests.
TFF_API long long tff_mlstm_workspace(int num_tokens, int num_requests, int H, int d, int dv) {
    const long long chunks = num_tokens / C + 2ll * num_requests;
    return chunks * H * ((long long)chunk_floats(d, dv) + NUMS);
}

// chunked != 0: chunk by chunk on the tensor cores, q, k and v rounded to bfloat16 (``workspace`` of tff_mlstm_workspace
// floats); else token by token in float32, and with norm_w (float32 [H*dv]) on to the mixer's output ``mixed`` [T, H*dv], where
// ``rows`` is proj again and ``clear`` sets the columns that were read to zero.  TFF_ERR_UNSUPPORTED when a head does not fit the form's shared memory.
TFF_API int tff_mlstm(const float* proj, int ld, int q_off, int k_off, int v_off, int i_off, int f_off, const float* gate_bias,
                      float cap, float q_scale, float* state, int num_slots, int slot_len, const int* q_start,
                      const int* pos_start, const int* slots, float* out, int num_requests, int H, int d, int dv, int chunked,
                      float* workspace, int num_tokens, float* rows, int g_off, const float* norm_w, float eps, void* mixed,
                      int mixed_is_bf16, int clear, cudaStream_t stream) {
    if (num_requests <= 0) return TFF_OK;
    if (norm_w && (chunked || !mixed || g_off < 0 || g_off + H * dv > ld || !(eps > 0.f) || (clear && !rows))) return TFF_ERR_BAD_ARGUMENT;
    if (!proj || !gate_bias || !state || !q_start || !pos_start || !slots || (!out && !norm_w) || H <= 0 || d <= 0 || dv <= 0 || !(cap > 0.f) ||
        q_off < 0 || k_off < 0 || v_off < 0 || i_off < 0 || f_off < 0 || q_off + H * d > ld || k_off + H * d > ld ||
        v_off + H * dv > ld || i_off + H > ld || f_off + H > ld || (slot_len & 3) ||
        (long long)slot_len < (long long)H * d * dv + (long long)H * d + H)
        return TFF_ERR_BAD_ARGUMENT;
    if (num_requests > 65535 || H > 65535) return TFF_ERR_UNSUPPORTED;
    const MlstmParams p{proj, ld, q_off, k_off, v_off, i_off, f_off, gate_bias, cap, q_scale, state, num_slots, slot_len,
                        q_start, pos_start, slots, out, H, d, dv, rows, g_off, norm_w, eps, mixed, mixed_is_bf16, clear};
    if (chunked) return launch_chunked(p, num_requests, workspace, num_tokens, stream);
    const bool vec = dv % 4 == 0 && ((uintptr_t)state & 15) == 0 && (H * d * dv) % 4 == 0;
    const bool single = num_tokens == num_requests && (long long)H * num_requests > 300;      // one token of many requests
    const int threads = single ? FEW : MANY, width = vec ? 4 : 1, groups = dv / width, lx = groups < threads ? groups : threads;
    const int ny = threads / lx;
    const bool keep = !single && groups <= threads && ny * ROWS >= d;
    const size_t smem = sizeof(float) * ((size_t)3 * d + dv + (size_t)ny * groups * width);
    if (smem > 48 * 1024) return TFF_ERR_UNSUPPORTED;
    const dim3 grid(H, num_requests);
#define TFF_STEP(VEC, KEEP, ST) return tff_launch_pdl(mlstm_step_kernel<VEC, KEEP, ST>, grid, dim3(ST), smem, stream, p)
    if (single) { if (vec) TFF_STEP(4, false, FEW); TFF_STEP(1, false, FEW); }
    if (vec) { if (keep) TFF_STEP(4, true, MANY); TFF_STEP(4, false, MANY); }
    if (keep) TFF_STEP(1, true, MANY);
    TFF_STEP(1, false, MANY);
#undef TFF_STEP
}

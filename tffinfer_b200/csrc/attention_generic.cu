// Causal grouped-query attention over the paged cache for flat token rows: one warp
// per (token, query head), any head size, any numbers of heads and groups, optional
// sliding window.  It is the attention of the true 32-bit path and takes every size
// the faster bfloat16 kernels refuse.
//
// For the token at position p of request b and query head h (kv head h / (nq/nkv),
// src/kernel/cuda/paged_flash_attention.cu:891-892):
//   s[n] = (q . k[n]) * scale for lo <= n <= p, lo = window ? max(0, p-window+1) : 0; with ``keep`` > 0 also for n < keep
//   s[n] = softcap * tanh(s[n] / softcap)                      when softcap > 0
//   out  = sum_n softmax(s)[n] * v[n]
// with the running-maximum ("online") softmax of the reference
// (paged_flash_attention.cu:696-792) in float32, over key blocks of 32 aligned to
// absolute positions.  The block boundaries depend on p and the window only, so a
// token's result does not depend on how the batch was cut or what else is in it.
// With ``sink`` the softmax has one more term in its denominator, a key that has no value and whose score (neither
// scaled nor capped) is sink_val[h], or 0 when sink_val is null: weights exp(s[n]) / (exp(sink) + sum exp(s)).  With ``gate`` (float32 [tokens, nq]) the head's output is multiplied by
// gate[t, h].  Keys have d elements and values dv; both lie in cache slots of dc >= max(d, dv) elements.
#include "common.cuh"
#include "attention_common.h"

namespace {

constexpr int WARPS = 4;

template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
attention_generic_kernel(const T* __restrict__ q_in, int row_stride,
                         const int* __restrict__ positions, const int* __restrict__ tok_req,
                         const int* __restrict__ block_table, int table_width,
                         const T* __restrict__ cache, KvLayout L, int layer,
                         T* __restrict__ out, int num_tokens, int nq, int nkv, int d, int dv,
                         float scale, int window, float softcap, int sink, const float* __restrict__ sink_val,
                         const float* __restrict__ gate, int keep) {
    extern __shared__ float smem[];            // WARPS * d floats: the warp's query row
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * WARPS + warp;
    if (item >= (long long)num_tokens * nq) return;
    const int t = (int)(item / nq), h = (int)(item % nq);
    const int kvh = h / (nq / nkv);
    const int p = positions[t];
    const int b = tok_req[t];
    const int* table = block_table + (size_t)b * table_width;
    float* q = smem + warp * d;
    const T* qrow = q_in + (size_t)t * row_stride + (size_t)h * d;
    for (int i = lane; i < d; i += 32) q[i] = to_f32<T>(qrow[i]);
    __syncwarp();

    const int lo = window > 0 ? max(0, p - window + 1) : 0;
    const int nd = (dv + 31) / 32;             // output dims per lane (<= 16 for dv <= 512)
    const int dc = L.head_dim;                 // elements of a cache slot
    float o[16];
#pragma unroll
    for (int j = 0; j < 16; ++j) o[j] = 0.f;
    // the sink is a key ahead of all others: its score starts the running maximum and the sum
    float m = sink ? (sink_val ? sink_val[h] : 0.f) : -INFINITY, l = sink ? 1.f : 0.f;
    const float inv_cap = softcap > 0.f ? 1.f / softcap : 0.f;

    const KeyWalk walk(keep, 32, lo / 32, p / 32);
    for (int w = 0; w < walk.count; ++w) {
        const int n = walk.block(w) * 32 + lane;
        const bool valid = n <= p && (n >= lo || n < keep);
        float s = -INFINITY;
        const T* vbase = nullptr;
        if (valid) {
            const int page = table[n / L.page_size];
            const T* kbase = cache + (size_t)page * L.page_stride + (size_t)layer * L.layer_stride +
                             (size_t)kvh * L.head_stride + (size_t)(n % L.page_size) * dc;
            vbase = kbase + L.kv_stride;
            float acc = 0.f;
            for (int i = 0; i < d; ++i) acc = fmaf(q[i], to_f32<T>(kbase[i]), acc);
            s = acc * scale;
            if (softcap > 0.f) s = softcap * tanhf(s * inv_cap);
        }
        const float bm = warp_max(s);          // at least lane with n == max(k0, lo) .. is valid
        const float m_new = fmaxf(m, bm);
        const float alpha = (m == -INFINITY) ? 0.f : expf(m - m_new);
        const float pr = valid ? expf(s - m_new) : 0.f;
        l = l * alpha + warp_sum(pr);
#pragma unroll
        for (int j = 0; j < 16; ++j) o[j] *= alpha;
        for (int kk = 0; kk < 32; ++kk) {
            const float pk = __shfl_sync(0xffffffffu, pr, kk);
            const unsigned long long vp = __shfl_sync(0xffffffffu, (unsigned long long)vbase, kk);
            if (vp == 0ull) continue;          // uniform across the warp
            const T* v = (const T*)vp;
#pragma unroll
            for (int j = 0; j < 16; ++j) {
                if (j < nd) {
                    const int i = j * 32 + lane;
                    if (i < dv) o[j] = fmaf(pk, to_f32<T>(v[i]), o[j]);
                }
            }
        }
        m = m_new;
    }
    const float inv = (gate ? gate[(size_t)t * nq + h] : 1.f) / l;
    T* orow = out + (size_t)t * nq * dv + (size_t)h * dv;
#pragma unroll
    for (int j = 0; j < 16; ++j) {
        if (j < nd) {
            const int i = j * 32 + lane;
            if (i < dv) orow[i] = from_f32<T>(o[j] * inv);
        }
    }
}

}  // namespace

// The general entry: keys of d and values of dv elements in cache slots of dc, score cap, sink, head gates.
TFF_API int tff_attention_generic_ext(
    const void* qkv, int is_bf16, int row_stride,
    const int* positions, const int* tok_req, const int* block_table, int table_width,
    const void* cache, int cache_layers, int layer, int page_size,
    void* out, int num_tokens, int nq, int nkv, int d, int dv, int dc, float scale, int window,
    float softcap, int sink, const float* sink_val, const float* gate, int keep, cudaStream_t stream) {
    if (num_tokens <= 0) return TFF_OK;
    if (nq <= 0 || nkv <= 0 || nq % nkv != 0 || d <= 0 || dv <= 0 || dc < d || dc < dv || page_size <= 0 || softcap < 0.f || keep < 0)
        return TFF_ERR_BAD_ARGUMENT;
    if (d > 512 || dv > 512) return TFF_ERR_UNSUPPORTED;
    if (window <= 0) keep = 0;
    const KvLayout L = make_kv_layout(cache_layers, nkv, page_size, dc);
    const long long items = (long long)num_tokens * nq;
    const unsigned blocks = (unsigned)((items + WARPS - 1) / WARPS);
    const size_t smem = (size_t)WARPS * d * sizeof(float);
    if (is_bf16)
        attention_generic_kernel<bf16><<<blocks, WARPS * 32, smem, stream>>>(
            (const bf16*)qkv, row_stride, positions, tok_req, block_table, table_width,
            (const bf16*)cache, L, layer, (bf16*)out, num_tokens, nq, nkv, d, dv, scale, window, softcap, sink, sink_val, gate, keep);
    else
        attention_generic_kernel<float><<<blocks, WARPS * 32, smem, stream>>>(
            (const float*)qkv, row_stride, positions, tok_req, block_table, table_width,
            (const float*)cache, L, layer, (float*)out, num_tokens, nq, nkv, d, dv, scale, window, softcap, sink, sink_val, gate, keep);
    return tff_launch_status();
}

TFF_API int tff_attention_generic(
    const void* qkv, int is_bf16, int row_stride,
    const int* positions, const int* tok_req, const int* block_table, int table_width,
    const void* cache, int cache_layers, int layer, int page_size,
    void* out, int num_tokens, int nq, int nkv, int d, float scale, int window, cudaStream_t stream) {
    return tff_attention_generic_ext(qkv, is_bf16, row_stride, positions, tok_req, block_table, table_width, cache,
                                     cache_layers, layer, page_size, out, num_tokens, nq, nkv, d, d, d, scale, window,
                                     0.f, 0, nullptr, nullptr, 0, stream);
}

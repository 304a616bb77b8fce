// Plain attention over the paged cache, one block per (token, query head),
// every step of the arithmetic in 32-bit.  It serves the 32-bit path for
// prefill and decode alike and any head size up to 256.
//
// The query at absolute position a sees key j iff j <= a and (window == 0 or
// a - j < window), or, with ``chunk`` > 0, iff j <= a and both lie in the same block of ``chunk`` positions; the first
// ``keep`` positions of a sequence are seen besides.  score = dot(q, k_j) / sqrt(hd) (divided after the product), or dot(q, k_j) * scale when a scale is
// given.  Values may have another size than keys (vd).  With ``sink`` the denominator holds one more term, exp(0 - max):
// a key of score zero that carries no value; with ``sink_vals`` the term is exp(sink_vals[head] - max), a number per head
// that is not scaled.  With ``softcap`` > 0 the scaled score s becomes softcap * tanh(s / softcap).  ``maps`` > 1: a key
// head's row in the cache holds that many keys side by side (hd numbers each) over one value; the query heads of a key
// head come map by map within each head, so query head h reads the key h % maps of key head h / (nh / nkv).  The result
// may be kept in float whatever the cache's type (TO), for a caller that goes on computing with it.
// Keys are walked in chunks of CHUNK positions aligned to absolute multiples of
// CHUNK with a running maximum and sum, so the order of every addition depends
// on the query's position alone: not on how the sequence was cut into steps,
// nor on what else is in the batch.
#include "common.cuh"

namespace {
constexpr int CHUNK = 256;
constexpr int THREADS = 128;
constexpr int MAX_HD = 256;

template <typename T, typename TO>
__global__ void __launch_bounds__(THREADS)
attn_simt_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache,
                 TO* __restrict__ out, const int* __restrict__ tok_seq, const int* __restrict__ tok_pos,
                 const int* __restrict__ block_table, int table_stride, int n_pages, int page, int nh, int nkv, int hd,
                 int vd, float scale, int sink, const float* __restrict__ sink_vals, int window, int chunk, int keep,
                 float softcap, int maps, int* __restrict__ status) {
    __shared__ float qs[MAX_HD];
    __shared__ float ps[CHUNK];
    __shared__ int pages[CHUNK];      // page id of each key of the chunk (or -1)
    __shared__ float scratch[33];
    const int n = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int seq = tok_seq[n], pos = tok_pos[n];
    const int kvh = h / (nh / nkv), map = h % maps;
    const VisibleKeys seen = visible_keys(pos, window, chunk, keep);
    const T* qrow = q + ((size_t)n * nh + h) * hd;
    for (int d = tid; d < hd; d += THREADS) qs[d] = to_f32(qrow[d]);
    const float root = sqrtf((float)hd);
    // the sink is a key of score zero (or of the head's own score) ahead of all others: the running maximum and sum start from it
    float m_run = sink ? (sink_vals ? sink_vals[h] : 0.f) : -INFINITY, l_run = sink ? 1.f : 0.f;
    float acc[MAX_HD / THREADS];
#pragma unroll
    for (int i = 0; i < MAX_HD / THREADS; i++) acc[i] = 0.f;
    __syncthreads();

    for (int c = seen.kept > 0 ? 0 : seen.lo / CHUNK; c <= pos / CHUNK; c++) {
        if (c * CHUNK >= seen.kept && c < seen.lo / CHUNK) c = seen.lo / CHUNK;     // nothing between the kept keys and the window
        const int j0 = c * CHUNK < seen.kept ? c * CHUNK : max(seen.lo, c * CHUNK), j1 = min(pos, c * CHUNK + CHUNK - 1);
        const int count = j1 - j0 + 1;
        // scores
        float local_max = -INFINITY;
        for (int t = tid; t < count; t += THREADS) {
            const int j = j0 + t;
            if (!seen.sees(j)) {                                     // a chunk that holds both kept keys and the window's first
                pages[t] = -1;
                ps[t] = -INFINITY;
                continue;
            }
            int pg = block_table[(size_t)seq * table_stride + j / page];
            if (pg < 0 || pg >= n_pages) {
                atomicOr(status, ESP_STATUS_BAD_INDEX);
                pg = -1;
            }
            pages[t] = pg;
            float s = -INFINITY;
            if (pg >= 0) {
                const T* krow = k_cache + ((((size_t)pg * nkv + kvh) * page + j % page) * maps + map) * hd;
                float dot = 0.f;
                for (int d = 0; d < hd; d++) dot = fmaf(qs[d], to_f32(krow[d]), dot);
                s = scale > 0.f ? dot * scale : dot / root;
                if (softcap > 0.f) s = softcap * tanhf(s / softcap);
            }
            ps[t] = s;
            local_max = fmaxf(local_max, s);
        }
        const float m_chunk = block_max(local_max, scratch);
        const float m_new = fmaxf(m_run, m_chunk);
        if (m_new == -INFINITY) continue;          // every key of the chunk was skipped as a bad index
        float local_sum = 0.f;
        for (int t = tid; t < count; t += THREADS) {
            const float p = expf(ps[t] - m_new);
            ps[t] = p;
            local_sum += p;
        }
        const float l_chunk = block_sum(local_sum, scratch);   // also orders the writes of ps before the reads below
        const float rescale = expf(m_run - m_new);
        l_run = l_run * rescale + l_chunk;
        m_run = m_new;
#pragma unroll
        for (int i = 0; i < MAX_HD / THREADS; i++) {
            const int d = tid + i * THREADS;
            if (d < vd) {
                float a = acc[i] * rescale;
                for (int t = 0; t < count; t++) {
                    const int pg = pages[t];
                    if (pg < 0) continue;
                    const int j = j0 + t;
                    a = fmaf(ps[t], to_f32(v_cache[(((size_t)pg * nkv + kvh) * page + j % page) * vd + d]), a);
                }
                acc[i] = a;
            }
        }
        __syncthreads();
    }
    TO* orow = out + ((size_t)n * nh + h) * vd;
#pragma unroll
    for (int i = 0; i < MAX_HD / THREADS; i++) {
        const int d = tid + i * THREADS;
        if (d < vd) orow[d] = from_f32<TO>(l_run > 0.f ? acc[i] / l_run : 0.f);
    }
}
}  // namespace

ESP_API int esp_attn_simt(const void* q, const void* k_cache, const void* v_cache, void* out, int is_bf16, int out_is_bf16,
                          const int* tok_seq, const int* tok_pos, const int* block_table, int table_stride, int n_pages,
                          int page, int n_tokens, int nh, int nkv, int hd, int vd, float scale, int sink,
                          const float* sink_vals, int window, int chunk, int keep, float softcap, int maps, int* status,
                          cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (vd <= 0) vd = hd;
    if (vd > MAX_HD || hd > MAX_HD || hd <= 0 || nkv <= 0 || nh % nkv != 0 || nh > 65535 || maps <= 0 || (nh / nkv) % maps != 0)
        return (int)cudaErrorInvalidValue;
    dim3 grid(n_tokens, nh);
#define ESP_SIMT(T, TO)                                                                                                    \
    attn_simt_kernel<T, TO><<<grid, THREADS, 0, stream>>>((const T*)q, (const T*)k_cache, (const T*)v_cache, (TO*)out, tok_seq, \
                                                          tok_pos, block_table, table_stride, n_pages, page, nh, nkv, hd, vd, \
                                                          scale, sink, sink_vals, window, chunk, keep, softcap, maps, status)
    if (is_bf16 && out_is_bf16) ESP_SIMT(bf16, bf16);
    else if (is_bf16) ESP_SIMT(bf16, float);
    else if (!out_is_bf16) ESP_SIMT(float, float);
    else return (int)cudaErrorInvalidValue;
#undef ESP_SIMT
    return esp_launch_status();
}

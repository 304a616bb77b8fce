// Linear attention with one fixed decay per head (bfloat16 engine): runs of many tokens in chunks on the tensor cores, runs of
// few tokens (decoding) token by token with the state in registers.
//
//     S_t = d S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t      per head; q, k, v = SiLU of the projections (float rows)
//
// A run of tokens is cut into chunks of C = 64.  With S the state ahead of a chunk, i and j counting its tokens from 0:
//
//     o_i = d^(i+1) S^T q_i + sum_(j <= i) d^(i-j) (q_i . k_j) v_j          S' = d^c S + sum_j d^(c-1-j) k_j v_j^T
//
// so only S is a chain over the chunks, and one multiply-add per entry and chunk at that.  Three kernels:
//
//   1. updates   U = sum_j d^(c-1-j) k_j v_j^T of every chunk and head (chunks in parallel), to scratch;
//   2. states    S' = d^c S + U, 32-bit, an entry of the state a thread quarter: from and to the sequence's state rows, every
//                chunk's S left where its U was;
//   3. outputs   of every chunk and head (chunks in parallel): scores, decayed and masked in 32-bit, times the values; plus
//                the queries times S.
//
// Products are mma.sync m16n8k16 with float accumulators.  Queries, keys of a score, values and a chunk's decayed scores are
// rounded to bfloat16; what the state is made of and what is read of it is not: a decayed key and an entry of S enter their
// products as the sum of two bfloat16 numbers.  The arithmetic is a few microseconds of the tensor cores' time at any size
// that the cache holds: what the kernels cost is the scratch's way through L2 and their loads, so the 5th-generation tensor
// cores (whose tiles of 128 would leave half the blocks) have nothing to win here.  The powers of d come from a table that
// the caller made in 64-bit.
#include "common.cuh"

namespace {
constexpr int C = 64, THREADS = 256, VT = 64;       // tokens of a chunk; value channels that a block works on at a time
constexpr int LDV = VT + 8, LDP = C + 8;            // row strides in shared memory: 16 bytes of padding against bank conflicts

__device__ __forceinline__ unsigned smem_at(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(unsigned (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_at(p)));
}
__device__ __forceinline__ void ldsm4_trans(unsigned (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_at(p)));
}
__device__ __forceinline__ void mma(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// fragments of a product's left operand kept [row][k] (16 rows from r0, 16 k from k0) ...
__device__ __forceinline__ const bf16* left_at(const bf16* t, int ld, int r0, int k0, int lane) {
    return t + (r0 + (lane & 15)) * ld + k0 + (lane >> 4) * 8;
}
// ... or kept [k][row] (read transposed)
__device__ __forceinline__ const bf16* left_trans_at(const bf16* t, int ld, int r0, int k0, int lane) {
    return t + (k0 + (lane & 7) + (lane >> 4) * 8) * ld + r0 + ((lane >> 3) & 1) * 8;
}
// fragments of two 8-column blocks of the right operand kept [column][k] ...
__device__ __forceinline__ const bf16* right_at(const bf16* t, int ld, int n0, int k0, int lane) {
    return t + (n0 + (lane & 7) + (lane >> 4) * 8) * ld + k0 + ((lane >> 3) & 1) * 8;
}
// ... or kept [k][column] (read transposed)
__device__ __forceinline__ const bf16* right_trans_at(const bf16* t, int ld, int n0, int k0, int lane) {
    return t + (k0 + (lane & 7) + ((lane >> 3) & 1) * 8) * ld + n0 + (lane >> 4) * 8;
}
__device__ __forceinline__ float silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
__device__ __forceinline__ float4 silu4(float4 v) { return make_float4(silu(v.x), silu(v.y), silu(v.z), silu(v.w)); }
__device__ __forceinline__ float low_part(float v) { return v - __bfloat162float(__float2bfloat16_rn(v)); }

struct ChunkList {
    const int *seq, *first, *seq_start;            // per chunk: its sequence, its first token among that sequence's new ones
};
struct Chunk {
    int row0, count;                               // first row among the packed tokens; tokens
};
__device__ __forceinline__ Chunk chunk_at(const ChunkList& l, int c) {
    const int s = l.seq[c], first = l.first[c];
    return Chunk{l.seq_start[s] + first, min(C, l.seq_start[s + 1] - l.seq_start[s] - first)};
}

// 64 rows of ``width`` channels, ``stride`` numbers apart, to shared memory [64][LD] as bfloat16 (rows from ``count`` on and
// channels past ``width`` up to W: zeros).  ACT: their SiLU.  scale (may be null): a factor per row; lo (may be null): what
// rounding left out, as a second tile.  A thread's loads go out several at a time.
template <int W, int LD, bool ACT>
__device__ __forceinline__ void stage(const float* src, long long stride, int count, int width, bf16* hi, bf16* lo, const float* scale) {
    constexpr int PIECES = W / 4, PER = 64 * PIECES / THREADS, BATCH = PER < 8 ? PER : 8;
    static_assert(64 * PIECES % THREADS == 0 && PER % BATCH == 0, "every thread stages the same number of pieces");
#pragma unroll
    for (int j0 = 0; j0 < PER; j0 += BATCH) {
        float4 v[BATCH];
#pragma unroll
        for (int j = 0; j < BATCH; j++) {
            const int i = threadIdx.x + (j0 + j) * THREADS, r = i / PIECES, c = (i % PIECES) * 4;
            v[j] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (r < count && c < width) v[j] = *reinterpret_cast<const float4*>(src + (size_t)r * stride + c);
        }
#pragma unroll
        for (int j = 0; j < BATCH; j++) {
            const int i = threadIdx.x + (j0 + j) * THREADS, r = i / PIECES, c = (i % PIECES) * 4;
            float4 s = ACT ? silu4(v[j]) : v[j];          // the SiLU of zero is zero
            if (scale) {
                const float f = scale[r];
                s.x *= f, s.y *= f, s.z *= f, s.w *= f;
            }
            Vec4<bf16>::store(hi + r * LD + c, s.x, s.y, s.z, s.w);
            if (lo) Vec4<bf16>::store(lo + r * LD + c, low_part(s.x), low_part(s.y), low_part(s.z), low_part(s.w));
        }
    }
}

// ---- 1. grid (chunks, heads, value tiles): scratch[chunk][head][v][k] = sum_j d^(c-1-j) k_j[k] v_j[v]
template <int KP>
__global__ void __launch_bounds__(THREADS)
linear_chunk_updates_kernel(const float* __restrict__ k, const float* __restrict__ v, long long ld, ChunkList list, int chunk0,
                            const float* __restrict__ powers, float* __restrict__ scratch, int K, int V) {
    constexpr int LDK = KP + 8, NB = KP / 16;       // a warp's share: 16 value channels x KP / 2 key channels, NB blocks of 8
    extern __shared__ __align__(16) unsigned char dyn[];
    bf16* k_hi = reinterpret_cast<bf16*>(dyn);      // [C][LDK]
    bf16* k_lo = k_hi + C * LDK;
    bf16* v_s = k_lo + C * LDK;                     // [C][LDV]
    __shared__ float fade[C];
    const int h = blockIdx.y, H = gridDim.y, v0 = blockIdx.z * VT, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const Chunk ch = chunk_at(list, chunk0 + blockIdx.x);
    if (threadIdx.x < C) fade[threadIdx.x] = threadIdx.x < ch.count ? powers[h * (C + 1) + ch.count - 1 - threadIdx.x] : 0.f;
    __syncthreads();
    stage<KP, LDK, true>(k + (size_t)ch.row0 * ld + h * K, ld, ch.count, K, k_hi, k_lo, fade);
    stage<VT, LDV, true>(v + (size_t)ch.row0 * ld + h * V + v0, ld, ch.count, V - v0, v_s, nullptr, nullptr);
    __syncthreads();
    const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * (KP / 2);
    float acc[NB][4];
#pragma unroll
    for (int b = 0; b < NB; b++)
#pragma unroll
        for (int i = 0; i < 4; i++) acc[b][i] = 0.f;
#pragma unroll
    for (int t = 0; t < C; t += 16) {
        unsigned a[4];
        ldsm4_trans(a, left_trans_at(v_s, LDV, m0, t, lane));
#pragma unroll
        for (int b = 0; b < NB; b += 2) {
            unsigned kh[4], kl[4];
            ldsm4_trans(kl, right_trans_at(k_lo, LDK, n0 + b * 8, t, lane));
            mma(acc[b], a, kl[0], kl[1]);
            mma(acc[b + 1], a, kl[2], kl[3]);
            ldsm4_trans(kh, right_trans_at(k_hi, LDK, n0 + b * 8, t, lane));
            mma(acc[b], a, kh[0], kh[1]);
            mma(acc[b + 1], a, kh[2], kh[3]);
        }
    }
    float* out = scratch + ((size_t)blockIdx.x * H + h) * V * K;
    const int g = lane >> 2, tg = lane & 3;
#pragma unroll
    for (int b = 0; b < NB; b++) {
        const int kc = n0 + b * 8 + tg * 2, va = v0 + m0 + g;
        if (kc >= K) continue;
        if (va < V) *reinterpret_cast<float2*>(out + (size_t)va * K + kc) = make_float2(acc[b][0], acc[b][1]);
        if (va + 8 < V) *reinterpret_cast<float2*>(out + (size_t)(va + 8) * K + kc) = make_float2(acc[b][2], acc[b][3]);
    }
}

// ---- 2. grid (pieces of the state, sequences): a thread owns four neighbouring key channels of a head's value channel
constexpr int AHEAD = 8;                            // updates in flight: their loads do not wait for the chain
__global__ void __launch_bounds__(128)
linear_chunk_states_kernel(float* __restrict__ scratch, float* __restrict__ state, long long state_stride,
                           const int* __restrict__ seq_slot, const int* __restrict__ chunk_start, ChunkList list, int chunk0,
                           int chunk1, const float* __restrict__ powers, int VK, int total) {
    const int piece = blockIdx.x * blockDim.x + threadIdx.x;
    if (piece * 4 >= total) return;
    const int b = blockIdx.y, h = piece * 4 / VK;
    const int c0 = max(chunk_start[b], chunk0), c1 = min(chunk_start[b + 1], chunk1);
    if (c0 >= c1) return;
    float4* own = reinterpret_cast<float4*>(state + (size_t)seq_slot[b] * state_stride) + piece;
    float4* u = reinterpret_cast<float4*>(scratch) + piece;
    const size_t step = (size_t)total / 4;
    const float* pw = powers + h * (C + 1);
    float4 S = *own;
    for (int c = c0; c < c1; c += AHEAD) {
        float4 next[AHEAD];
        float f[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; i++)
            if (c + i < c1) {
                next[i] = u[(size_t)(c + i - chunk0) * step];
                f[i] = pw[chunk_at(list, c + i).count];
            }
#pragma unroll
        for (int i = 0; i < AHEAD; i++)
            if (c + i < c1) {
                u[(size_t)(c + i - chunk0) * step] = S;
                S.x = fmaf(f[i], S.x, next[i].x), S.y = fmaf(f[i], S.y, next[i].y);
                S.z = fmaf(f[i], S.z, next[i].z), S.w = fmaf(f[i], S.w, next[i].w);
            }
    }
    *own = S;
}

// ---- 3. grid (chunks, heads): scratch[chunk][head][v][k] holds the state ahead of the chunk
template <int KP>
__global__ void __launch_bounds__(THREADS)
linear_chunk_outputs_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, long long ld,
                            ChunkList list, int chunk0, const float* __restrict__ powers, const float* __restrict__ scratch,
                            float* __restrict__ out, int K, int V) {
    constexpr int LDK = KP + 8;
    extern __shared__ __align__(16) unsigned char dyn[];
    bf16* q_s = reinterpret_cast<bf16*>(dyn);       // [C][LDK]
    bf16* s_hi = q_s + C * LDK;                     // [VT][LDK]: the tile of S; the chunk's keys before that
    bf16* s_lo = s_hi + VT * LDK;
    bf16* p_s = s_lo + VT * LDK;                    // [C][LDP] decayed scores
    bf16* v_s = p_s + C * LDP;                      // [C][LDV]
    __shared__ float pw[C + 1];
    const int h = blockIdx.y, H = gridDim.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int g = lane >> 2, tg = lane & 3;
    const Chunk ch = chunk_at(list, chunk0 + blockIdx.x);
    if (threadIdx.x <= C) pw[threadIdx.x] = powers[h * (C + 1) + threadIdx.x];
    stage<KP, LDK, true>(q + (size_t)ch.row0 * ld + h * K, ld, ch.count, K, q_s, nullptr, nullptr);
    stage<KP, LDK, true>(k + (size_t)ch.row0 * ld + h * K, ld, ch.count, K, s_hi, nullptr, nullptr);
    __syncthreads();
    const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 32;   // a warp's share of a 64 x 64 tile: 16 tokens x 32 columns
    const int ta = m0 + g, tb = ta + 8;                      // the lane's two tokens
    float acc[4][4];
    auto clear = [&] {
#pragma unroll
        for (int b = 0; b < 4; b++)
#pragma unroll
            for (int i = 0; i < 4; i++) acc[b][i] = 0.f;
    };
    clear();
#pragma unroll
    for (int kk = 0; kk < KP; kk += 16) {
        unsigned a[4];
        ldsm4(a, left_at(q_s, LDK, m0, kk, lane));
#pragma unroll
        for (int b = 0; b < 4; b += 2) {
            unsigned kf[4];
            ldsm4(kf, right_at(s_hi, LDK, n0 + b * 8, kk, lane));
            mma(acc[b], a, kf[0], kf[1]);
            mma(acc[b + 1], a, kf[2], kf[3]);
        }
    }
#pragma unroll
    for (int b = 0; b < 4; b++) {
        const int j = n0 + b * 8 + tg * 2;
        auto w = [&](int t, int key, float s) { return key <= t ? s * pw[t - key] : 0.f; };
        *reinterpret_cast<__nv_bfloat162*>(p_s + ta * LDP + j) = __floats2bfloat162_rn(w(ta, j, acc[b][0]), w(ta, j + 1, acc[b][1]));
        *reinterpret_cast<__nv_bfloat162*>(p_s + tb * LDP + j) = __floats2bfloat162_rn(w(tb, j, acc[b][2]), w(tb, j + 1, acc[b][3]));
    }
    const float* S = scratch + ((size_t)blockIdx.x * H + h) * V * K;
    for (int v0 = 0; v0 < V; v0 += VT) {
        __syncthreads();                            // the keys (or the tile before) have been read, the scores are written
        stage<KP, LDK, false>(S + (size_t)v0 * K, K, V - v0, K, s_hi, s_lo, nullptr);
        stage<VT, LDV, true>(v + (size_t)ch.row0 * ld + h * V + v0, ld, ch.count, V - v0, v_s, nullptr, nullptr);
        __syncthreads();
        clear();
#pragma unroll
        for (int kk = 0; kk < KP; kk += 16) {
            unsigned a[4];
            ldsm4(a, left_at(q_s, LDK, m0, kk, lane));
#pragma unroll
            for (int b = 0; b < 4; b += 2) {
                unsigned sf[4];
                ldsm4(sf, right_at(s_lo, LDK, n0 + b * 8, kk, lane));
                mma(acc[b], a, sf[0], sf[1]);
                mma(acc[b + 1], a, sf[2], sf[3]);
                ldsm4(sf, right_at(s_hi, LDK, n0 + b * 8, kk, lane));
                mma(acc[b], a, sf[0], sf[1]);
                mma(acc[b + 1], a, sf[2], sf[3]);
            }
        }
        const float fa = pw[ta + 1], fb = pw[tb + 1];
#pragma unroll
        for (int b = 0; b < 4; b++) acc[b][0] *= fa, acc[b][1] *= fa, acc[b][2] *= fb, acc[b][3] *= fb;
#pragma unroll
        for (int t = 0; t < C; t += 16) {
            if (t > m0 + 15) break;                 // keys behind the warp's last token weigh nothing
            unsigned a[4];
            ldsm4(a, left_at(p_s, LDP, m0, t, lane));
#pragma unroll
            for (int b = 0; b < 4; b += 2) {
                unsigned vf[4];
                ldsm4_trans(vf, right_trans_at(v_s, LDV, n0 + b * 8, t, lane));
                mma(acc[b], a, vf[0], vf[1]);
                mma(acc[b + 1], a, vf[2], vf[3]);
            }
        }
#pragma unroll
        for (int b = 0; b < 4; b++) {
            const int vc = v0 + n0 + b * 8 + tg * 2;
            if (vc >= V) continue;
            float* o = out + (size_t)ch.row0 * H * V + (size_t)h * V + vc;
            if (ta < ch.count) *reinterpret_cast<float2*>(o + (size_t)ta * H * V) = make_float2(acc[b][0], acc[b][1]);
            if (tb < ch.count) *reinterpret_cast<float2*>(o + (size_t)tb * H * V) = make_float2(acc[b][2], acc[b][3]);
        }
    }
}

// ---- runs of few tokens: grid (sequences, heads, value tiles).  A warp owns STEP_ROWS value channels of a head, a lane four
// key channels of each (KL times); the state stays in registers over the run.  It was written by an earlier step, so its loads
// do not wait for the kernel before this one.
constexpr int STEP_ROWS = 4, STEP_WARPS = 4;
template <int KL>
__global__ void __launch_bounds__(32 * STEP_WARPS)
linear_steps_kernel(const float* __restrict__ q, const float* __restrict__ k, const float* __restrict__ v, long long ld,
                    const float* __restrict__ decay, const float* __restrict__ rest, float* __restrict__ state,
                    long long state_stride, const int* __restrict__ seq_start, const int* __restrict__ seq_slot,
                    float* __restrict__ out, int K, int V) {
    pdl_trigger();
    const int b = blockIdx.x, h = blockIdx.y, H = gridDim.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int v0 = (blockIdx.z * STEP_WARPS + warp) * STEP_ROWS;
    const int row0 = seq_start[b], row1 = seq_start[b + 1];
    const float d = decay[h], d_rest = rest[h];
    float* own = state + (size_t)seq_slot[b] * state_stride + (size_t)h * V * K + (size_t)v0 * K + lane * 4;
    const float4 none = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 S[STEP_ROWS][KL];
#pragma unroll
    for (int r = 0; r < STEP_ROWS; r++)
#pragma unroll
        for (int l = 0; l < KL; l++)
            S[r][l] = v0 + r < V && lane * 4 + l * 128 < K ? *reinterpret_cast<const float4*>(own + r * K + l * 128) : none;
    pdl_wait();
    const float* q_now = behind_wait(q);
    const float* k_now = behind_wait(k);
    const float* v_now = behind_wait(v);
    for (int t = row0; t < row1; t++) {
        float4 qv[KL], kv[KL];
#pragma unroll
        for (int l = 0; l < KL; l++) {
            const int c = lane * 4 + l * 128;
            qv[l] = c < K ? silu4(*reinterpret_cast<const float4*>(q_now + t * ld + h * K + c)) : none;
            kv[l] = c < K ? silu4(*reinterpret_cast<const float4*>(k_now + t * ld + h * K + c)) : none;
        }
        float o[STEP_ROWS];
#pragma unroll
        for (int r = 0; r < STEP_ROWS; r++) {
            const float val = v0 + r < V ? silu(v_now[t * ld + h * V + v0 + r]) : 0.f;
            o[r] = 0.f;
#pragma unroll
            for (int l = 0; l < KL; l++) {
                float4& s = S[r][l];
                s.x = fmaf(d, s.x, fmaf(d_rest, s.x, kv[l].x * val)), s.y = fmaf(d, s.y, fmaf(d_rest, s.y, kv[l].y * val));
                s.z = fmaf(d, s.z, fmaf(d_rest, s.z, kv[l].z * val)), s.w = fmaf(d, s.w, fmaf(d_rest, s.w, kv[l].w * val));
                o[r] = fmaf(s.w, qv[l].w, fmaf(s.z, qv[l].z, fmaf(s.y, qv[l].y, fmaf(s.x, qv[l].x, o[r]))));
            }
        }
#pragma unroll
        for (int r = 0; r < STEP_ROWS; r++) o[r] = warp_sum(o[r]);
        if (lane < STEP_ROWS && v0 + lane < V) out[(size_t)t * H * V + h * V + v0 + lane] = lane == 0 ? o[0] : lane == 1 ? o[1] : lane == 2 ? o[2] : o[3];
    }
    static_assert(STEP_ROWS == 4, "a lane each writes the outputs");
#pragma unroll
    for (int r = 0; r < STEP_ROWS; r++)
#pragma unroll
        for (int l = 0; l < KL; l++)
            if (v0 + r < V && lane * 4 + l * 128 < K) *reinterpret_cast<float4*>(own + r * K + l * 128) = S[r][l];
}

template <int KP>
int run(const float* q, const float* k, const float* v, long long ld, ChunkList list, const int* chunk_start, int n_chunks,
        int chunks_at_once, const float* powers, float* scratch, float* state, long long state_stride, const int* seq_slot,
        float* out, int n_seqs, int H, int K, int V, cudaStream_t stream) {
    constexpr size_t smem_u = (size_t)(2 * C * (KP + 8) + C * LDV) * sizeof(bf16);
    constexpr size_t smem_o = (size_t)((C + 2 * VT) * (KP + 8) + C * LDP + C * LDV) * sizeof(bf16);
    static bool raised = false;
    if (!raised) {
        cudaError_t e = cudaFuncSetAttribute(linear_chunk_updates_kernel<KP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_u);
        if (e == cudaSuccess)
            e = cudaFuncSetAttribute(linear_chunk_outputs_kernel<KP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_o);
        if (e != cudaSuccess) return (int)e;
        raised = true;
    }
    const int total = H * V * K;
    for (int c0 = 0; c0 < n_chunks; c0 += chunks_at_once) {
        const int n = n_chunks - c0 < chunks_at_once ? n_chunks - c0 : chunks_at_once;
        linear_chunk_updates_kernel<KP><<<dim3(n, H, (V + VT - 1) / VT), THREADS, smem_u, stream>>>(k, v, ld, list, c0, powers, scratch,
                                                                                                    K, V);
        linear_chunk_states_kernel<<<dim3((total / 4 + 127) / 128, n_seqs), 128, 0, stream>>>(
            scratch, state, state_stride, seq_slot, chunk_start, list, c0, c0 + n, powers, V * K, total);
        linear_chunk_outputs_kernel<KP><<<dim3(n, H), THREADS, smem_o, stream>>>(q, k, v, ld, list, c0, powers, scratch, out, K, V);
    }
    return esp_launch_status();
}
}  // namespace

// q, k [rows, H * K] and v [rows, H * V]: float, before their SiLU, rows ``ld`` numbers apart; chunk_seq / chunk_first: every
// chunk of up to 64 new tokens (sequence, first token among that sequence's new ones), in order of the sequences;
// chunk_start [n_seqs + 1]: the sequences' ranges in that list; powers [H, 65]: d_h^0 .. d_h^64; scratch:
// min(n_chunks, chunks_at_once) * H * V * K floats; state: a head's block [V][K] floats at h * V * K in the slot's row; out
// [rows, H * V] float.  K and V multiples of 4 (and of ld and the state's stride), K at most 256; every buffer 16-byte aligned.
ESP_API int esp_linear_attn_chunks(const float* q, const float* k, const float* v, long long ld, const int* chunk_seq,
                                   const int* chunk_first, const int* chunk_start, const int* seq_start, const int* seq_slot,
                                   const float* powers, float* scratch, int chunks_at_once, float* state, long long state_stride,
                                   float* out, int n_chunks, int n_seqs, int H, int K, int V, cudaStream_t stream) {
    if (n_chunks <= 0) return 0;
    const size_t ptrs = (size_t)q | (size_t)k | (size_t)v | (size_t)scratch | (size_t)state | (size_t)out;
    if (K <= 0 || V <= 0 || K > 256 || K % 4 || V % 4 || ld % 4 || state_stride % 4 || (ptrs & 15) || chunks_at_once <= 0 || H <= 0 ||
        H > 65535 || n_seqs > 65535 || (long long)H * V * K >= (1ll << 31))
        return (int)cudaErrorInvalidValue;
    const ChunkList list{chunk_seq, chunk_first, seq_start};
#define ESP_CHUNKS(KP)                                                                                                        \
    return run<KP>(q, k, v, ld, list, chunk_start, n_chunks, chunks_at_once, powers, scratch, state, state_stride, seq_slot, out, \
                   n_seqs, H, K, V, stream)
    if (K <= 32) ESP_CHUNKS(32);
    if (K <= 64) ESP_CHUNKS(64);
    if (K <= 128) ESP_CHUNKS(128);
    ESP_CHUNKS(256);
#undef ESP_CHUNKS
}

// The same for runs of few tokens.  decay, rest [H]: the decay and what 32-bit leaves out of it.  Sizes as above.
ESP_API int esp_linear_attn_steps(const float* q, const float* k, const float* v, long long ld, const float* decay, const float* rest,
                                  float* state, long long state_stride, const int* seq_start, const int* seq_slot, float* out,
                                  int n_seqs, int H, int K, int V, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    const size_t ptrs = (size_t)q | (size_t)k | (size_t)v | (size_t)state;
    if (K <= 0 || V <= 0 || K > 256 || K % 4 || V % 4 || ld % 4 || state_stride % 4 || (ptrs & 15) || H <= 0 || H > 65535)
        return (int)cudaErrorInvalidValue;
    const dim3 grid(n_seqs, H, (V + STEP_ROWS * STEP_WARPS - 1) / (STEP_ROWS * STEP_WARPS));
    if (K <= 128)
        esp_launch_pdl(ESP_PDL_SMALL, linear_steps_kernel<1>, grid, dim3(32 * STEP_WARPS), 0, stream, q, k, v, ld, decay, rest, state,
                       state_stride, seq_start, seq_slot, out, K, V);
    else
        esp_launch_pdl(ESP_PDL_SMALL, linear_steps_kernel<2>, grid, dim3(32 * STEP_WARPS), 0, stream, q, k, v, ld, decay, rest, state,
                       state_stride, seq_start, seq_slot, out, K, V);
    return esp_launch_status();
}

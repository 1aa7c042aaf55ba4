// Linear attention with a fading memory: per head a matrix S [D, DV] in float32 from zero and, per token,
//
//   channel decays     S <- diag(alpha_t) S + k v^T ;  o = S^T (q D^-1/2),  alpha_t = sigmoid(z_t + b)^(1 / tau) per key channel
//                      (Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training")
//   constant decay     S <- decay_h S + silu(k) silu(v)^T ;  o = S^T silu(q)
//                      (Qin et al., "Lightning Attention-2: A Free Lunch for Handling Unlimited Sequence Lengths in Large
//                      Language Models")
//
// Three forms of the same recurrence:
//
//   decay_step    a single token of every request (decoding in bfloat16 models): one pass over S.
//   decay_scan    one token after the other (memory_scan.cuh): short portions, and the whole 32-bit path, where a token's
//                 output must not depend on how its prompt was cut.
//   decay_chunks  long portions, chunks of 64 tokens side by side. With g_t the running product of decays inside a chunk (from
//                 its first token on, so g <= 1), G the chunk's whole product and S_c the memory before the chunk:
//                     o_i = (q_i g_i)^T S_c + sum_{j <= i} ((q_i g_i) . (k_j / g_j)) v_j
//                     S_(c+1) = G S_c + sum_j (k_j G / g_j) v_j^T
//                 Four launches: the running logarithms of the decays (channel decays only), every chunk's own sum, the
//                 memories at the chunks' starts (memory_scan.cuh: pieces_combine), the outputs. All of it in float32 on the FMA
//                 pipe (the memory, the decays and what enters them are float32 by the designs' own rule, so the tensor cores,
//                 which would round the operands, are left out), as register-tiled products from shared memory.
//                 1 / g_j can overflow where a channel forgets nearly everything within a chunk: a CTA whose chunk has a
//                 channel with g below e^-60 forms its scores with exp(log g_i - log g_j) per channel instead, which only
//                 costs time. A constant decay never divides: decay^(i - j) is taken from a table of powers.
#include "memory_scan.cuh"

namespace stride {

constexpr int kChunk = 64;              // tokens a chunk
constexpr int kChunkCols = 128;         // columns of S a CTA works on
constexpr int kSumCols = 64;            // the same in the kernel of the chunks' own sums
constexpr int kChunkThreads = 256;
constexpr int kLd = kChunk + 4;         // row stride of the transposed tiles: 16-byte reads, stores without bank conflicts
constexpr float kSafeLog = -60.f;

struct ChunkArgs {
    const void* q;          // [tokens, ld], head h at column h * D
    const void* k;
    const void* v;          // head h at column h * DV
    int ld, in_bf16;
    float* cum;             // channel decays: [tokens, H * D], the running logarithm of the decays inside the chunk
    const float* bias;      // channel decays: [H * D]
    const float* powers;    // constant decay: [H, kChunk + 1], decay^n
    float q_scale, inv_tau;
    float* o;               // [tokens, H * DV]
    float* piece_s;         // [seqs * max_pieces, H, D, DV]
    float* piece_p;         // [seqs * max_pieces, H, D]
    const int32_t* q_start;
    const int32_t* q_len;
    int H, D, DV, max_pieces;
    int vec;                // bfloat16 rows that can be read in packs of 8
};

// z -> running sums of log(sigmoid(z + b)) / tau over the chunk's tokens, in place. One thread a (head, channel).
static __global__ void __launch_bounds__(128)
chunk_decay_kernel(const ChunkArgs p) {
    pdl_trigger();
    pdl_wait();
    const int z = blockIdx.y, seq = z / p.max_pieces, first = (z % p.max_pieces) * kChunk;
    const int nt = min(p.q_len[seq] - first, kChunk);
    const int c = blockIdx.x * blockDim.x + threadIdx.x, HD = p.H * p.D;
    if (nt <= 0 || c >= HD) return;
    float* at = p.cum + static_cast<size_t>(p.q_start[seq] + first) * HD + c;
    const float b = p.bias[c];
    float sum = 0.f, lost = 0.f;        // Kahan's sum: differences of these sums are the exponents of whole decays
    for (int t0 = 0; t0 < nt; t0 += 8) {
        float l[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) l[u] = t0 + u < nt ? at[static_cast<size_t>(t0 + u) * HD] : 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u) l[u] = log_sigmoid_f(l[u] + b) * p.inv_tau;
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (t0 + u < nt) {
                const float y = __fadd_rn(l[u], -lost), next = __fadd_rn(sum, y);
                lost = __fadd_rn(__fadd_rn(next, -sum), -y);
                sum = next;
                at[static_cast<size_t>(t0 + u) * HD] = sum;
            }
    }
}

// Eight neighbouring values of a row of the projection.
__device__ __forceinline__ void unpack8(const uint4& r, float* v) {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(h[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ const uint4* row8(const void* base, size_t at) {
    return reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(base) + at);
}

// The values of a chunk [kChunk][COLS] from column col0 on into shared memory, zeros beyond the head; rows from nt on are left out.
template <int COLS, int RULE>
__device__ __forceinline__ void stage_values(const ChunkArgs& p, float* vs, size_t row0, int nt, int h, int col0) {
    if (p.vec) {
        constexpr int PACKS = kChunk * COLS / 8 / kChunkThreads;        // packs a thread
        uint4 raw[PACKS];
#pragma unroll
        for (int n = 0; n < PACKS; ++n) {
            const int idx = n * kChunkThreads + threadIdx.x, j = idx / (COLS / 8), c = (idx % (COLS / 8)) * 8;
            raw[n] = j < nt && col0 + c < p.DV ? *row8(p.v, (row0 + j) * p.ld + h * p.DV + col0 + c) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int n = 0; n < PACKS; ++n) {
            const int idx = n * kChunkThreads + threadIdx.x, j = idx / (COLS / 8), c = (idx % (COLS / 8)) * 8;
            float v[8];
            unpack8(raw[n], v);
            if (RULE == kConstantDecay) {
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = silu_quick(v[e]);
            }
            float4* dst = reinterpret_cast<float4*>(vs + j * COLS + c);
            dst[0] = make_float4(v[0], v[1], v[2], v[3]);
            dst[1] = make_float4(v[4], v[5], v[6], v[7]);
        }
        return;
    }
    for (int idx = threadIdx.x; idx < nt * COLS; idx += kChunkThreads) {
        const int j = idx / COLS, c = idx - j * COLS;
        float v = 0.f;
        if (col0 + c < p.DV) {
            v = load_any(p.v, (row0 + j) * p.ld + h * p.DV + col0 + c, p.in_bf16);
            if (RULE == kConstantDecay) v = silu_f(v);
        }
        vs[idx] = v;
    }
}

// piece_s[z, h] = sum_j (k_j G / g_j) v_j^T, piece_p[z, h] = G. DP: D padded. Grid (tiles of kSumCols columns, heads, chunks).
template <int DP, int RULE>
__global__ void __launch_bounds__(kChunkThreads)
chunk_sum_kernel(const ChunkArgs p) {
    constexpr int PASS_ROWS = DP < 128 ? DP : 128, R = PASS_ROWS / 16;      // rows of S a half warp holds at a time
    extern __shared__ __align__(16) float smem[];
    float* ks = smem;                       // [kChunk][DP]
    float* vs = smem + kChunk * DP;         // [kChunk][kSumCols]
    pdl_trigger();
    const int z = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * kSumCols;
    const int seq = z / p.max_pieces, first = (z % p.max_pieces) * kChunk;
    const int nt = min(p.q_len[seq] - first, kChunk);
    if (nt <= 0) return;
    pdl_wait();
    const int D = p.D, DV = p.DV, HD = p.H * D;
    const size_t row0 = static_cast<size_t>(p.q_start[seq] + first);
    const float* powers = RULE == kConstantDecay ? p.powers + h * (kChunk + 1) : nullptr;
    const float* cum = RULE == kChannelDecay ? p.cum + row0 * HD + h * D : nullptr;
    if (p.vec) {
        constexpr int PACKS = kChunk * DP / 8 / kChunkThreads > 0 ? kChunk * DP / 8 / kChunkThreads : 1;
        uint4 raw[PACKS];
#pragma unroll
        for (int n = 0; n < PACKS; ++n) {
            const int idx = n * kChunkThreads + threadIdx.x, j = idx / (DP / 8), d = (idx % (DP / 8)) * 8;
            raw[n] = j < nt && d < D ? *row8(p.k, (row0 + j) * p.ld + h * D + d) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int n = 0; n < PACKS; ++n) {
            const int idx = n * kChunkThreads + threadIdx.x, j = idx / (DP / 8), d = (idx % (DP / 8)) * 8;
            float k[8];
            unpack8(raw[n], k);
            if (RULE == kConstantDecay) {
                const float f = j < nt ? powers[nt - 1 - j] : 0.f;
#pragma unroll
                for (int e = 0; e < 8; ++e) k[e] = silu_quick(k[e]) * f;
            } else if (j < nt && d < D) {
                const float4* end = reinterpret_cast<const float4*>(cum + static_cast<size_t>(nt - 1) * HD + d);
                const float4* own = reinterpret_cast<const float4*>(cum + static_cast<size_t>(j) * HD + d);
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const float4 a = end[u], b = own[u];
                    k[4 * u] *= expf(a.x - b.x);
                    k[4 * u + 1] *= expf(a.y - b.y);
                    k[4 * u + 2] *= expf(a.z - b.z);
                    k[4 * u + 3] *= expf(a.w - b.w);
                }
            }
            if (j < kChunk) {
                float4* dst = reinterpret_cast<float4*>(ks + j * DP + d);
                dst[0] = make_float4(k[0], k[1], k[2], k[3]);
                dst[1] = make_float4(k[4], k[5], k[6], k[7]);
            }
        }
    } else {
        for (int idx = threadIdx.x; idx < nt * DP; idx += kChunkThreads) {
            const int j = idx / DP, d = idx - j * DP;
            float k = 0.f;
            if (d < D) {
                k = load_any(p.k, (row0 + j) * p.ld + h * D + d, p.in_bf16);
                k = RULE == kConstantDecay ? silu_f(k) * powers[nt - 1 - j]
                                           : k * expf(cum[static_cast<size_t>(nt - 1) * HD + d] - cum[static_cast<size_t>(j) * HD + d]);
            }
            ks[idx] = k;
        }
    }
    stage_values<kSumCols, RULE>(p, vs, row0, nt, h, col0);
    if (blockIdx.x == 0)
        for (int d = threadIdx.x; d < D; d += kChunkThreads)
            p.piece_p[(static_cast<size_t>(z) * p.H + h) * D + d] =
                RULE == kConstantDecay ? powers[nt] : expf(cum[static_cast<size_t>(nt - 1) * HD + d]);
    __syncthreads();
    const int warp = threadIdx.x >> 5, cg = (threadIdx.x & 15) * 4, half = (threadIdx.x >> 4) & 1;
    float* out = p.piece_s + (static_cast<size_t>(z) * p.H + h) * D * DV;
    for (int pass = 0; pass < DP / PASS_ROWS; ++pass) {
        const int r0 = pass * PASS_ROWS + (2 * warp + half) * R;
        float acc[R][4];
#pragma unroll
        for (int r = 0; r < R; ++r) acc[r][0] = acc[r][1] = acc[r][2] = acc[r][3] = 0.f;
#pragma unroll 4
        for (int j = 0; j < nt; ++j) {
            const float4 b = *reinterpret_cast<const float4*>(vs + j * kSumCols + cg);
            float a[R];
            if constexpr (R >= 4) {
#pragma unroll
                for (int r = 0; r < R; r += 4) {
                    const float4 a4 = *reinterpret_cast<const float4*>(ks + j * DP + r0 + r);
                    a[r] = a4.x; a[r + 1] = a4.y; a[r + 2] = a4.z; a[r + 3] = a4.w;
                }
            } else {
#pragma unroll
                for (int r = 0; r < R; ++r) a[r] = ks[j * DP + r0 + r];
            }
#pragma unroll
            for (int r = 0; r < R; ++r) {
                acc[r][0] = fmaf(a[r], b.x, acc[r][0]);
                acc[r][1] = fmaf(a[r], b.y, acc[r][1]);
                acc[r][2] = fmaf(a[r], b.z, acc[r][2]);
                acc[r][3] = fmaf(a[r], b.w, acc[r][3]);
            }
        }
#pragma unroll
        for (int r = 0; r < R; ++r) {
            if (r0 + r >= D) continue;
            float* dst = out + static_cast<size_t>(r0 + r) * DV + col0 + cg;
            if (DV % 4 == 0) {
                if (col0 + cg < DV) *reinterpret_cast<float4*>(dst) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (col0 + cg + e < DV) dst[e] = acc[r][e];
            }
        }
    }
}

// Between the two: piece_s becomes the memory at every chunk's start, the state the memory after the last one. As
// pieces_combine_kernel, with four neighbouring columns a thread.
static __global__ void __launch_bounds__(256)
chunk_combine_kernel(float4* __restrict__ piece_s, const float* __restrict__ piece_p, float* __restrict__ state, long long state_stride,
                     const int32_t* __restrict__ q_len, const int32_t* __restrict__ state_slot, int H, int D, int DV, int max_pieces) {
    pdl_trigger();
    const int seq = blockIdx.y;
    const int len = q_len[seq];
    const int entry = blockIdx.x * blockDim.x + threadIdx.x, entries = H * D * DV / 4;
    if (len <= 0 || entry >= entries) return;
    pdl_wait();
    const int row = entry * 4 / DV;                                      // h * D + i
    float4* S_g = reinterpret_cast<float4*>(state + static_cast<size_t>(state_slot[seq]) * state_stride) + entry;
    float4 S = *S_g;
    const int pieces = (len + kChunk - 1) / kChunk;
    constexpr int AHEAD = 8;        // chunks whose loads are in flight together
    for (int c0 = 0; c0 < pieces; c0 += AHEAD) {
        float4 own[AHEAD];
        float decay[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u)
            if (c0 + u < pieces) {
                const size_t z = static_cast<size_t>(seq) * max_pieces + c0 + u;
                own[u] = piece_s[z * entries + entry];
                decay[u] = piece_p[z * H * D + row];
            }
#pragma unroll
        for (int u = 0; u < AHEAD; ++u)
            if (c0 + u < pieces) {
                piece_s[(static_cast<size_t>(seq) * max_pieces + c0 + u) * entries + entry] = S;
                S.x = fmaf(decay[u], S.x, own[u].x);
                S.y = fmaf(decay[u], S.y, own[u].y);
                S.z = fmaf(decay[u], S.z, own[u].z);
                S.w = fmaf(decay[u], S.w, own[u].w);
            }
    }
    *S_g = S;
}

// Outputs of a chunk from the memory at its start (piece_s by now). Grid (tiles of kChunkCols columns, heads, chunks).
template <int DP>
__host__ __device__ constexpr int chunk_second_floats() { return DP * kLd > kChunk * kChunkCols ? DP * kLd : kChunk * kChunkCols; }
template <int DP>
__host__ __device__ constexpr int chunk_out_floats() { return DP * kLd + chunk_second_floats<DP>() + kChunk * kLd; }

template <int DP, int RULE>
__global__ void __launch_bounds__(kChunkThreads, DP <= 128 ? 2 : 1)
chunk_out_kernel(const ChunkArgs p) {
    constexpr int SLAB = 64 < DP ? 64 : DP;         // rows of S staged at a time
    constexpr int SLAB_PACKS = SLAB * kChunkCols / 4 / kChunkThreads;
    extern __shared__ __align__(16) float smem[];
    float* qT = smem;                               // [DP][kLd]: column i is token i's query (times g_i)
    float* kT = qT + DP * kLd;                      // [DP][kLd]; later slabs of S [SLAB][kChunkCols], then the values [kChunk][kChunkCols]
    float* aT = kT + chunk_second_floats<DP>();     // [kChunk j][kLd i]: scores
    pdl_trigger();
    const int z = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * kChunkCols;
    const int seq = z / p.max_pieces, first = (z % p.max_pieces) * kChunk;
    const int nt = min(p.q_len[seq] - first, kChunk);
    if (nt <= 0) return;
    pdl_wait();
    const int D = p.D, DV = p.DV, HD = p.H * D;
    const size_t row0 = static_cast<size_t>(p.q_start[seq] + first);
    const float* powers = RULE == kConstantDecay ? p.powers + h * (kChunk + 1) : nullptr;
    const float* cum = RULE == kChannelDecay ? p.cum + row0 * HD + h * D : nullptr;
    bool safe = true;
    if (RULE == kChannelDecay) {
        int low = 0;
        for (int d = threadIdx.x; d < D; d += kChunkThreads) low |= cum[static_cast<size_t>(nt - 1) * HD + d] < kSafeLog;
        safe = !__syncthreads_or(low);
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (p.vec) {
        // a warp takes packs of 8 channels, its lanes 32 neighbouring tokens: the transposed stores hit 32 banks
        constexpr int PACKS = DP / 8 * 2 / 8;       // (pack, half of the tokens) pairs a warp
        uint4 rq[PACKS], rk[PACKS];
#pragma unroll
        for (int n = 0; n < PACKS; ++n) {
            const int item = n * 8 + warp, d = (item >> 1) * 8, i = (item & 1) * 32 + lane;
            const bool ok = i < nt && d < D;
            const size_t at = (row0 + i) * p.ld + h * D + d;
            rq[n] = ok ? *row8(p.q, at) : make_uint4(0, 0, 0, 0);
            rk[n] = ok ? *row8(p.k, at) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int n = 0; n < PACKS; ++n) {
            const int item = n * 8 + warp, d = (item >> 1) * 8, i = (item & 1) * 32 + lane;
            float q[8], k[8];
            unpack8(rq[n], q);
            unpack8(rk[n], k);
            if (RULE == kConstantDecay) {
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    q[e] = silu_quick(q[e]);
                    k[e] = silu_quick(k[e]);
                }
            } else if (i < nt && d < D) {
                const float4* own = reinterpret_cast<const float4*>(cum + static_cast<size_t>(i) * HD + d);
                const float4 c0 = own[0], c1 = own[1];
                const float c[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    q[e] *= safe ? p.q_scale * expf(c[e]) : p.q_scale;
                    if (safe) k[e] *= expf(-c[e]);
                }
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                qT[(d + e) * kLd + i] = q[e];
                kT[(d + e) * kLd + i] = k[e];
            }
        }
    } else {
        // lanes of a warp: 8 neighbouring channels of 4 neighbouring tokens
        for (int idx = threadIdx.x; idx < kChunk * DP; idx += kChunkThreads) {
            const int sub = idx & 31, blk = idx >> 5;
            const int d = (blk % (DP / 8)) * 8 + (sub & 7), i = (blk / (DP / 8)) * 4 + (sub >> 3);
            float q = 0.f, k = 0.f;
            if (d < D && i < nt) {
                const size_t at = (row0 + i) * p.ld + h * D + d;
                q = load_any(p.q, at, p.in_bf16);
                k = load_any(p.k, at, p.in_bf16);
                if (RULE == kConstantDecay) {
                    q = silu_f(q);
                    k = silu_f(k);
                } else {
                    q *= p.q_scale;
                    if (safe) {
                        const float c = cum[static_cast<size_t>(i) * HD + d];
                        q *= expf(c);
                        k *= expf(-c);
                    }
                }
            }
            qT[d * kLd + i] = q;
            kT[d * kLd + i] = k;
        }
    }
    // the first rows of S travel while the scores are worked out
    const float* S = p.piece_s + (static_cast<size_t>(z) * p.H + h) * D * DV;
    const bool s_vec = DV % 4 == 0;
    float4 ahead[SLAB_PACKS];
    auto fetch_slab = [&](int d0) {
#pragma unroll
        for (int n = 0; n < SLAB_PACKS; ++n) {
            const int idx = n * kChunkThreads + threadIdx.x, d = d0 + idx / (kChunkCols / 4), c = col0 + (idx % (kChunkCols / 4)) * 4;
            ahead[n] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (d < D && c < DV) {
                const float* at = S + static_cast<size_t>(d) * DV + c;
                if (s_vec) {
                    ahead[n] = *reinterpret_cast<const float4*>(at);
                } else {
                    ahead[n].x = at[0];
                    if (c + 1 < DV) ahead[n].y = at[1];
                    if (c + 2 < DV) ahead[n].z = at[2];
                    if (c + 3 < DV) ahead[n].w = at[3];
                }
            }
        }
    };
    fetch_slab(0);
    __syncthreads();
    {   // scores: thread (ty, tx) tokens i = 4 ty .. + 3 against j = 4 tx .. + 3
        const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
        float a[4][4];
#pragma unroll
        for (int e = 0; e < 4; ++e) a[e][0] = a[e][1] = a[e][2] = a[e][3] = 0.f;
        if (RULE == kConstantDecay || safe) {
            if (tx <= ty) {
#pragma unroll 8
                for (int d = 0; d < DP; ++d) {
                    const float4 q4 = *reinterpret_cast<const float4*>(qT + d * kLd + 4 * ty);
                    const float4 k4 = *reinterpret_cast<const float4*>(kT + d * kLd + 4 * tx);
                    const float qv[4] = {q4.x, q4.y, q4.z, q4.w}, kv[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e)
#pragma unroll
                        for (int f = 0; f < 4; ++f) a[e][f] = fmaf(qv[e], kv[f], a[e][f]);
                }
            }
        } else if (tx <= ty) {
            for (int d = 0; d < D; ++d) {
                float ci[4], cj[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    ci[e] = 4 * ty + e < nt ? cum[static_cast<size_t>(4 * ty + e) * HD + d] : 0.f;
                    cj[e] = 4 * tx + e < nt ? cum[static_cast<size_t>(4 * tx + e) * HD + d] : 0.f;
                }
#pragma unroll
                for (int e = 0; e < 4; ++e)
#pragma unroll
                    for (int f = 0; f < 4; ++f)
                        if (4 * tx + f <= 4 * ty + e) a[e][f] = fmaf(qT[d * kLd + 4 * ty + e] * expf(ci[e] - cj[f]), kT[d * kLd + 4 * tx + f], a[e][f]);
            }
        }
#pragma unroll
        for (int f = 0; f < 4; ++f) {
            float w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int n = 4 * ty + e - (4 * tx + f);
                w[e] = n < 0 ? 0.f : RULE == kConstantDecay ? a[e][f] * powers[n] : a[e][f];
            }
            *reinterpret_cast<float4*>(aT + (4 * tx + f) * kLd + 4 * ty) = make_float4(w[0], w[1], w[2], w[3]);
        }
    }
    __syncthreads();
    if (RULE == kChannelDecay && !safe) {
        for (int idx = threadIdx.x; idx < kChunk * DP; idx += kChunkThreads) {
            const int i = idx % kChunk, d = idx / kChunk;
            if (d < D && i < nt) qT[d * kLd + i] *= expf(cum[static_cast<size_t>(i) * HD + d]);
        }
    }
    // outputs: warp w tokens 8 w .. + 7, lane columns 4 lane .. + 3
    float acc[8][4];
#pragma unroll
    for (int r = 0; r < 8; ++r) acc[r][0] = acc[r][1] = acc[r][2] = acc[r][3] = 0.f;
    auto step = [&](const float* a_row, const float* b_row) {
        const float4 lo = *reinterpret_cast<const float4*>(a_row), hi = *reinterpret_cast<const float4*>(a_row + 4);
        const float4 b = *reinterpret_cast<const float4*>(b_row);
        const float a[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            acc[r][0] = fmaf(a[r], b.x, acc[r][0]);
            acc[r][1] = fmaf(a[r], b.y, acc[r][1]);
            acc[r][2] = fmaf(a[r], b.z, acc[r][2]);
            acc[r][3] = fmaf(a[r], b.w, acc[r][3]);
        }
    };
    for (int d0 = 0; d0 < DP && d0 < D; d0 += SLAB) {
#pragma unroll
        for (int n = 0; n < SLAB_PACKS; ++n) *reinterpret_cast<float4*>(kT + (n * kChunkThreads + threadIdx.x) * 4) = ahead[n];
        __syncthreads();
        if (d0 + SLAB < D) fetch_slab(d0 + SLAB);
#pragma unroll 4
        for (int d = 0; d < SLAB; ++d) step(qT + (d0 + d) * kLd + 8 * warp, kT + d * kChunkCols + 4 * lane);
        __syncthreads();
    }
    if (RULE == kConstantDecay) {
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            const float f = powers[8 * warp + r + 1];
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[r][e] *= f;
        }
    }
    stage_values<kChunkCols, RULE>(p, kT, row0, nt, h, col0);
    __syncthreads();
    const int last = min(nt, 8 * warp + 8);         // later tokens have no weight in this warp's rows
#pragma unroll 4
    for (int j = 0; j < last; ++j) step(aT + j * kLd + 8 * warp, kT + j * kChunkCols + 4 * lane);
#pragma unroll
    for (int r = 0; r < 8; ++r) {
        const int i = 8 * warp + r;
        if (i >= nt) break;
        float* dst = p.o + ((row0 + i) * p.H + h) * DV + col0 + 4 * lane;
        if (s_vec) {
            if (col0 + 4 * lane < DV) *reinterpret_cast<float4*>(dst) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (col0 + 4 * lane + e < DV) dst[e] = acc[r][e];
        }
    }
}

// A single token of every request: one pass over S, which is all there is to do. A warp reads whole rows of up to 128 columns, the
// eight warps of a CTA take every eighth row; their shares of S^T q meet in shared memory. Grid (tiles of 128 columns, heads, requests).
template <int RULE>
__global__ void __launch_bounds__(kChunkThreads)
decay_step_kernel(const ScanArgs p) {
    __shared__ float s_q[256], s_k[256], s_w[256];
    __shared__ __align__(16) float red[8][kChunkCols];
    pdl_trigger();
    const int seq = blockIdx.z, h = blockIdx.y, col = blockIdx.x * kChunkCols + 4 * (threadIdx.x & 31);
    if (p.q_len[seq] <= 0) return;
    pdl_wait();
    const int D = p.D, DV = p.DV, warp = threadIdx.x >> 5;
    const size_t row = static_cast<size_t>(p.q_start[seq]);
    float* S_g = p.state + static_cast<size_t>(p.state_slot[seq]) * p.state_stride + static_cast<size_t>(h) * D * DV + col;
    constexpr int AHEAD = 16;
    float4 S[AHEAD];
    const bool live = col < DV;
#pragma unroll
    for (int u = 0; u < AHEAD; ++u)
        if (live && warp + 8 * u < D) S[u] = *reinterpret_cast<const float4*>(S_g + static_cast<size_t>(warp + 8 * u) * DV);
    const int d = threadIdx.x;
    if (d < D) {
        const size_t at = row * p.lda + h * D + d;
        const float q = load_any(p.a, at, p.in_bf16), k = load_any(p.k, at, p.in_bf16);
        s_q[d] = RULE == kConstantDecay ? silu_f(q) : q * p.q_scale;
        s_k[d] = RULE == kConstantDecay ? silu_f(k) : k;
        s_w[d] = RULE == kConstantDecay ? p.fade[h] : expm1f(log_sigmoid_f(p.w[row * p.H * D + h * D + d] + p.w0[h * D + d]) * p.inv_tau);
    }
    float v[4] = {0.f, 0.f, 0.f, 0.f}, acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (live) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            v[e] = load_any(p.v, row * p.ldv + h * DV + col + e, p.in_bf16);
            if (RULE == kConstantDecay) v[e] = silu_f(v[e]);
        }
    }
    __syncthreads();
    for (int d0 = 0; d0 < D; d0 += 8 * AHEAD) {
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int i = d0 + warp + 8 * u;
            if (live && i < D) {
                const float w = s_w[i], k = s_k[i], q = s_q[i];
                float x[4] = {S[u].x, S[u].y, S[u].z, S[u].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    x[e] = fmaf(k, v[e], fmaf(w, x[e], x[e]));
                    acc[e] = fmaf(q, x[e], acc[e]);
                }
                *reinterpret_cast<float4*>(S_g + static_cast<size_t>(i) * DV) = make_float4(x[0], x[1], x[2], x[3]);
            }
        }
#pragma unroll
        for (int u = 0; u < AHEAD; ++u) {
            const int i = d0 + 8 * AHEAD + warp + 8 * u;
            if (live && i < D) S[u] = *reinterpret_cast<const float4*>(S_g + static_cast<size_t>(i) * DV);
        }
    }
    *reinterpret_cast<float4*>(&red[warp][4 * (threadIdx.x & 31)]) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    __syncthreads();
    if (threadIdx.x < kChunkCols && blockIdx.x * kChunkCols + threadIdx.x < DV) {
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) sum += red[w][threadIdx.x];
        p.o[(row * p.H + h) * DV + blockIdx.x * kChunkCols + threadIdx.x] = sum;
    }
}

template <typename... A>
cudaError_t more_shared_memory(void (*kernel)(A...), int bytes) {
    return bytes > 48 * 1024 ? cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) : cudaSuccess;
}

template <int DP, int RULE>
int launch_chunks(const ChunkArgs& p, float* state, long long state_stride, const int32_t* state_slot, int num_seqs, cudaStream_t stream) {
    const int zs = num_seqs * p.max_pieces;
    const dim3 grid((p.DV + kChunkCols - 1) / kChunkCols, p.H, zs), block(kChunkThreads);
    const dim3 sum_grid((p.DV + kSumCols - 1) / kSumCols, p.H, zs);
    constexpr int sum_bytes = (kChunk * DP + kChunk * kSumCols) * 4, out_bytes = chunk_out_floats<DP>() * 4;
    cudaError_t e = more_shared_memory(chunk_sum_kernel<DP, RULE>, sum_bytes);
    if (e == cudaSuccess) e = more_shared_memory(chunk_out_kernel<DP, RULE>, out_bytes);
    if (e != cudaSuccess) return static_cast<int>(e);
    if (RULE == kChannelDecay) stride::launch(chunk_decay_kernel, dim3((p.H * p.D + 127) / 128, zs), dim3(128), 0, stream, p);
    stride::launch(chunk_sum_kernel<DP, RULE>, sum_grid, block, sum_bytes, stream, p);
    if (p.DV % 4 == 0 && state_stride % 4 == 0 && reinterpret_cast<uintptr_t>(state) % 16 == 0)
        stride::launch(chunk_combine_kernel, dim3((p.H * p.D * p.DV / 4 + 255) / 256, num_seqs), dim3(256), 0, stream,
                       reinterpret_cast<float4*>(p.piece_s), static_cast<const float*>(p.piece_p), state, state_stride, p.q_len, state_slot, p.H,
                       p.D, p.DV, p.max_pieces);
    else
        stride::launch(pieces_combine_kernel, dim3((p.H * p.D * p.DV + 255) / 256, num_seqs), dim3(256), 0, stream, p.piece_s,
                       static_cast<const float*>(p.piece_p), state, state_stride, p.q_len, state_slot, p.H, p.D, p.DV, kChunk, p.max_pieces);
    stride::launch(chunk_out_kernel<DP, RULE>, grid, block, out_bytes, stream, p);
    return STRIDE_LAUNCH_STATUS();
}

template <int RULE>
int dispatch_chunks(const ChunkArgs& p, float* state, long long state_stride, const int32_t* state_slot, int num_seqs, cudaStream_t stream) {
    if (p.D <= 32) return launch_chunks<32, RULE>(p, state, state_stride, state_slot, num_seqs, stream);
    if (p.D <= 64) return launch_chunks<64, RULE>(p, state, state_stride, state_slot, num_seqs, stream);
    if (p.D <= 128) return launch_chunks<128, RULE>(p, state, state_stride, state_slot, num_seqs, stream);
    if (p.D <= 256) return launch_chunks<256, RULE>(p, state, state_stride, state_slot, num_seqs, stream);
    return STRIDE_UNSUPPORTED;
}

inline ScanArgs decay_args(const void* q, const void* k, const void* v, int ld, const float* logit, const float* bias, const float* fade,
                           float q_scale, float inv_tau, float* o, float* state, long long state_stride, const int32_t* q_start,
                           const int32_t* q_len, const int32_t* state_slot, int H, int D, int DV, int dtype) {
    ScanArgs p = {};
    p.a = q;
    p.k = k;
    p.v = v;
    p.lda = p.ldv = ld;
    p.w = logit;
    p.w0 = bias;
    p.fade = fade;
    p.q_scale = q_scale;
    p.inv_tau = inv_tau;
    p.o = o;
    p.state = state;
    p.state_stride = state_stride;
    p.q_start = q_start;
    p.q_len = q_len;
    p.state_slot = state_slot;
    p.H = H;
    p.group = 1;
    p.D = D;
    p.DV = DV;
    p.in_bf16 = dtype == STRIDE_DTYPE_BF16 ? 1 : 0;
    return p;
}

}  // namespace stride

using namespace stride;

extern "C" {

// One token after the other. q, k [tokens, ld] with head h at column h * D, v with head h at column h * DV, all in the compute
// type. fade (constant decay): [H] float32, the decay minus one; null: channel decays from logit [tokens, H * D] and bias
// [H * D], float32. o [tokens, H * DV] float32; state: S of head h at h * D * DV floats into a slot's row.
int stride_decay_scan(const void* q, const void* k, const void* v, int ld, const float* logit, const float* bias, const float* fade,
                      float q_scale, float inv_tau, float* o, float* state, long long state_stride, const int32_t* q_start,
                      const int32_t* q_len, const int32_t* state_slot, int num_seqs, int H, int D, int DV, int dtype, cudaStream_t stream) {
    if (num_seqs < 0 || H <= 0 || D <= 0 || DV <= 0 || (!fade && (!logit || !bias))) return STRIDE_BAD_ARGUMENT;
    if (state_stride < static_cast<long long>(H) * D * DV) return STRIDE_BAD_ARGUMENT;
    if (dtype != STRIDE_DTYPE_F32 && dtype != STRIDE_DTYPE_BF16) return STRIDE_BAD_ARGUMENT;
    if (num_seqs > 65535 || H > 65535) return STRIDE_UNSUPPORTED;
    if (num_seqs == 0) return 0;
    const ScanArgs p = decay_args(q, k, v, ld, logit, bias, fade, q_scale, inv_tau, o, state, state_stride, q_start, q_len, state_slot, H, D, DV, dtype);
    return fade ? launch_scan<kConstantDecay>(p, num_seqs, stream) : launch_scan<kChannelDecay>(p, num_seqs, stream);
}

// The same for requests that bring exactly one token each (q_len 0: none); returns -2 for what it does not take (values in
// widths that are no multiple of 4, rows off 16-byte boundaries): decay_scan runs everything.
int stride_decay_step(const void* q, const void* k, const void* v, int ld, const float* logit, const float* bias, const float* fade,
                      float q_scale, float inv_tau, float* o, float* state, long long state_stride, const int32_t* q_start,
                      const int32_t* q_len, const int32_t* state_slot, int num_seqs, int H, int D, int DV, int dtype, cudaStream_t stream) {
    if (num_seqs < 0 || H <= 0 || D <= 0 || DV <= 0 || (!fade && (!logit || !bias))) return STRIDE_BAD_ARGUMENT;
    if (state_stride < static_cast<long long>(H) * D * DV) return STRIDE_BAD_ARGUMENT;
    if (dtype != STRIDE_DTYPE_F32 && dtype != STRIDE_DTYPE_BF16) return STRIDE_BAD_ARGUMENT;
    if (num_seqs > 65535 || H > 65535 || D > 256 || DV % 4 || state_stride % 4 || reinterpret_cast<uintptr_t>(state) % 16) return STRIDE_UNSUPPORTED;
    if (num_seqs == 0) return 0;
    ScanArgs p = decay_args(q, k, v, ld, logit, bias, fade, q_scale, inv_tau, o, state, state_stride, q_start, q_len, state_slot, H, D, DV, dtype);
    const dim3 grid((DV + kChunkCols - 1) / kChunkCols, H, num_seqs);
    stride::launch(fade ? decay_step_kernel<kConstantDecay> : decay_step_kernel<kChannelDecay>, grid, dim3(kChunkThreads), 0, stream, p);
    return STRIDE_LAUNCH_STATUS();
}

// Chunk by chunk. powers (constant decay): [H, 65] float32, decay^0 .. decay^64; null: channel decays, whose logits are
// overwritten. scratch: float32, num_seqs * max_pieces * H * D * (DV + 1), max_pieces = ceil(longest portion / 64).
int stride_decay_chunks(const void* q, const void* k, const void* v, int ld, float* logit, const float* bias, const float* powers,
                        float q_scale, float inv_tau, float* o, float* state, long long state_stride, const int32_t* q_start,
                        const int32_t* q_len, const int32_t* state_slot, int num_seqs, int H, int D, int DV, int dtype, int max_pieces,
                        float* scratch, cudaStream_t stream) {
    if (num_seqs < 0 || H <= 0 || D <= 0 || DV <= 0 || max_pieces <= 0 || !scratch || (!powers && (!logit || !bias))) return STRIDE_BAD_ARGUMENT;
    if (state_stride < static_cast<long long>(H) * D * DV) return STRIDE_BAD_ARGUMENT;
    if (dtype != STRIDE_DTYPE_F32 && dtype != STRIDE_DTYPE_BF16) return STRIDE_BAD_ARGUMENT;
    if (static_cast<long long>(num_seqs) * max_pieces > 65535 || H > 65535 || reinterpret_cast<uintptr_t>(scratch) % 16) return STRIDE_UNSUPPORTED;
    if (num_seqs == 0) return 0;
    ChunkArgs p = {};
    p.q = q;
    p.k = k;
    p.v = v;
    p.ld = ld;
    p.in_bf16 = dtype == STRIDE_DTYPE_BF16 ? 1 : 0;
    p.cum = logit;
    p.bias = bias;
    p.powers = powers;
    p.q_scale = q_scale;
    p.inv_tau = inv_tau;
    p.o = o;
    p.piece_s = scratch;
    p.piece_p = scratch + static_cast<size_t>(num_seqs) * max_pieces * H * D * DV;
    p.q_start = q_start;
    p.q_len = q_len;
    p.H = H;
    p.D = D;
    p.DV = DV;
    p.max_pieces = max_pieces;
    auto aligned = [](const void* x) { return reinterpret_cast<uintptr_t>(x) % 16 == 0; };
    p.vec = p.in_bf16 && D % 8 == 0 && DV % 8 == 0 && ld % 8 == 0 && aligned(q) && aligned(k) && aligned(v) && (powers || aligned(logit));
    return powers ? dispatch_chunks<kConstantDecay>(p, state, state_stride, state_slot, num_seqs, stream)
                  : dispatch_chunks<kChannelDecay>(p, state, state_stride, state_slot, num_seqs, stream);
}

}  // extern "C"

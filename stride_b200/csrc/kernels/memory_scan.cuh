// The scan shared by the mixers whose memory is a matrix per head (linear_recurrence.cu, decay_memory.cu, state_space.cu): a head's S [D, DV]
// in registers, one token after the other, any of the rules below; and the pass between pieces of a long portion.
#pragma once

#include "common.cuh"

namespace stride {

enum MemoryRule {
    kDeltaRule = 0,         // S <- diag(1 + w) S ; u = beta (v - S^T k) ; S <- S + k u^T ; o = S^T a
    kBonusMemory = 1,       // o = (S + diag(bonus) k v^T)^T a ; S <- diag(exp(-exp(w + w0))) S + k v^T
    kChannelDecay = 2,      // S <- diag(sigmoid(w + w0)^(1 / tau)) S + k v^T ; o = q_scale S^T a
    kConstantDecay = 3,     // S <- (1 + fade) S + silu(k) silu(v)^T ; o = S^T silu(a)
    kTokenDecay = 4,        // d = softplus(beta + dt_bias), S <- exp(-exp(a_log) d) S + d k v^T ; o = S^T a + skip v (a number a head and token)
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
// The same by the hardware's exponential and quotient: a few units in the last place of float32.
__device__ __forceinline__ float silu_quick(float z) { return __fdividef(z, 1.f + __expf(-z)); }

__device__ __forceinline__ float load_any(const void* p, size_t i, int is_bf16) {
    return is_bf16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(p)[i]) : static_cast<const float*>(p)[i];
}
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// --------------------------------------------------------------------------------------------------------- scans
constexpr int kScanThreads = 128;

struct ScanArgs {
    const void* a;          // queries (delta) / receptance (memory with bonus): [tokens, lda], head h at column (h / group) * D
    const void* k;          // keys, the same layout
    const float* w;         // [tokens, H * D]: the decay minus one (delta), its double logarithm before w0 (bonus rule), or the
                            // logit before w0 whose sigmoid to the power 1 / tau is the decay (channel decays)
    const void* v;          // values [tokens, ldv], head h at column h * DV
    const float* beta;      // [tokens, H] (delta); [tokens, ld_beta]: step sizes before bias and softplus (token decay); or null
    const float* w0;        // [H * D] added to w before exp(-exp(.)) (bonus rule) or the sigmoid (channel decays), or null
    const float* bonus;     // [H * D] (bonus rule) or null
    const float* fade;      // [H] (constant decay): the head's decay minus one
    float q_scale, inv_tau; // channel decays: what queries are multiplied by, and 1 / tau
    float* o;               // [tokens, H * DV] float32
    float* state;           // [slots, state_stride]; S of head h at h * D * DV
    long long state_stride;
    const int32_t* q_start;
    const int32_t* q_len;
    const int32_t* state_slot;
    int lda, ldv, H, group, D, DV, in_bf16;
    const float* dt_bias;   // [H] each (token decay)
    const float* a_log;
    const float* skip;
    int ld_beta;
    // the convolution's tail (delta rule; taps 0: none): the last taps - 1 rows of proj's first C columns
    const void* proj;
    int ld_proj, C, taps, proj_bf16;
    long long tail_off;
    // pieces (mode 0: none, a request's tokens in one chain). A piece is `piece` consecutive tokens of a request; grid z is
    // request * max_pieces + piece. Mode 1 runs every piece from a zero memory, writes no output, and leaves the piece's
    // memory in piece_s [z, H, D, DV] and the product of its decays in piece_p [z, H, D]; mode 2 runs every piece from
    // piece_s (by then the memory at the piece's start), writes the outputs and leaves the state alone.
    // init (mode 1): 1 starts every column from zero, 2 from the unit matrix (column j holds a one in row j): with no values
    // (v null) the memory of a piece then ends as the matrix that carries any memory across the piece.
    int mode, piece, max_pieces, init;
    float* piece_s;
    float* piece_p;
};

// LANES lanes share a column, each with R of its rows (R a multiple of 4): D <= LANES * R. A thread works on NC columns
// at once (COLS apart), CHUNK tokens are staged at a time. One token follows the other and a warp issues in order, so what
// sets the pace of a prompt is the chain of dependent instructions a token costs a warp (shared-memory reads, the sums,
// the shuffles), not the amount of arithmetic: the rows are spread over as many lanes as the head size allows, and the NC
// columns of a thread are independent chains that fill one another's waits (they also share the reads of k, q and the decay).
// PIECES false: the one chain only (mode 0), with nothing of the pieces' bookkeeping in its loop.
template <int LANES, int R, int NC, int CHUNK, int RULE, bool PIECES>      // RULE: see MemoryRule
__global__ void __launch_bounds__(kScanThreads)
scan_kernel(const ScanArgs p) {
    // Launched without programmatic dependent launch (launch_alone): no trigger, and nothing to wait for.
    const int mode = PIECES ? p.mode : 0;
    constexpr int DP = R * LANES;                           // rows with padding
    constexpr int THREADS = kScanThreads;
    constexpr int COLS = THREADS / LANES;                   // columns of one pass over the threads
    constexpr int CTA_COLS = COLS * NC;                     // columns of this CTA
    constexpr int ROW_ITEMS = CHUNK * DP / THREADS;         // entries of each [chunk, DP] array a thread fetches
    constexpr int V_ITEMS = (CHUNK * CTA_COLS + THREADS - 1) / THREADS;
    static_assert(R % 4 == 0 && (CHUNK * DP) % THREADS == 0 && CHUNK <= THREADS, "chunks are shared out evenly");
    // two buffers: while the tokens of one chunk are worked through, the next chunk's inputs are on their way from
    // global memory into registers; they are stored (the decay's exponentials applied) when the chunk is done
    __shared__ __align__(16) float s_a[2][CHUNK][DP], s_k[2][CHUNK][DP], s_w[2][CHUNK][DP];
    __shared__ float s_v[2][CHUNK][CTA_COLS], s_beta[2][CHUNK];
    __shared__ __align__(16) float s_bonus[DP], s_w0[DP];
    const int seq = mode ? blockIdx.z / p.max_pieces : blockIdx.z, h = blockIdx.y;
    const int first = mode ? (blockIdx.z % p.max_pieces) * p.piece : 0;         // this CTA's tokens of the request: [first, len)
    const int len = mode ? min(p.q_len[seq], first + p.piece) : p.q_len[seq];
    if (len <= first) return;
    const int start = p.q_start[seq];
    const int il = threadIdx.x & (LANES - 1), jc = threadIdx.x / LANES;
    const int j0 = blockIdx.x * CTA_COLS + jc;              // this thread's columns: j0 + c * COLS
    const int D = p.D, DV = p.DV, H = p.H;
    const int hk = h / p.group;
    float* S_g = mode ? p.piece_s + (static_cast<size_t>(blockIdx.z) * H + h) * D * DV
                        : p.state + static_cast<size_t>(p.state_slot[seq]) * p.state_stride + static_cast<size_t>(h) * D * DV;
    // lane il of a column's lanes holds rows 4 LANES g + 4 il + e (g < R / 4, e < 4) in S[.][4 g + e]: four neighbouring rows
    // are one 16-byte read of shared memory, and the lanes read consecutive 16 bytes
    auto row_of = [&](int r) { return 4 * LANES * (r >> 2) + 4 * il + (r & 3); };
    float S[NC][R];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int i = row_of(r), j = j0 + c * COLS;
            S[c][r] = mode == 1 ? ((p.init == 2 && i == j && i < D) ? 1.f : 0.f)
                                  : ((i < D && j < DV) ? S_g[static_cast<size_t>(i) * DV + j] : 0.f);
        }
    float decayed[R];           // mode 1: the product of the decays of this thread's rows over the piece
#pragma unroll
    for (int r = 0; r < R; ++r) decayed[r] = 1.f;
    if (RULE == kBonusMemory || RULE == kChannelDecay)
        for (int i = threadIdx.x; i < DP; i += blockDim.x) {
            if (RULE == kBonusMemory) s_bonus[i] = i < D ? p.bonus[h * D + i] : 0.f;
            s_w0[i] = i < D ? p.w0[h * D + i] : 0.f;
        }
    const float fade = RULE == kConstantDecay ? p.fade[h] : 0.f;
    const float rate = RULE == kTokenDecay ? expf(p.a_log[h]) : 0.f, dt_bias = RULE == kTokenDecay ? p.dt_bias[h] : 0.f;
    const float skip = RULE == kTokenDecay ? p.skip[h] : 0.f;

    float fa[ROW_ITEMS], fk[ROW_ITEMS], fw[ROW_ITEMS], fv[V_ITEMS], fb = 0.f;
    auto fetch = [&](int c0) {          // the chunk from token c0 on, into registers (zeros past the request's end)
#pragma unroll
        for (int n = 0; n < ROW_ITEMS; ++n) {
            const int idx = n * THREADS + threadIdx.x;
            const int tt = idx / DP, i = idx - tt * DP;
            fa[n] = fk[n] = fw[n] = 0.f;
            if (c0 + tt < len && i < D) {
                const size_t row = static_cast<size_t>(start + c0 + tt);
                fa[n] = load_any(p.a, row * p.lda + hk * D + i, p.in_bf16);
                fk[n] = load_any(p.k, row * p.lda + hk * D + i, p.in_bf16);
                if (RULE != kConstantDecay && RULE != kTokenDecay) fw[n] = p.w[row * H * D + h * D + i];
            }
        }
#pragma unroll
        for (int n = 0; n < V_ITEMS; ++n) {
            const int idx = n * THREADS + threadIdx.x;
            const int tt = idx / CTA_COLS, c = idx - tt * CTA_COLS;
            const int col = blockIdx.x * CTA_COLS + c;
            fv[n] = ((!PIECES || p.v != nullptr) && tt < CHUNK && c0 + tt < len && col < DV)
                        ? load_any(p.v, static_cast<size_t>(start + c0 + tt) * p.ldv + h * DV + col, p.in_bf16) : 0.f;
        }
        if (RULE == 0 && threadIdx.x < CHUNK)
            fb = c0 + threadIdx.x < len ? p.beta[static_cast<size_t>(start + c0 + threadIdx.x) * H + h] : 0.f;
        if (RULE == kTokenDecay && threadIdx.x < CHUNK)
            fb = c0 + threadIdx.x < len ? p.beta[static_cast<size_t>(start + c0 + threadIdx.x) * p.ld_beta + h] : 0.f;
    };
    auto stash = [&](int buf) {
#pragma unroll
        for (int n = 0; n < ROW_ITEMS; ++n) {
            const int idx = n * THREADS + threadIdx.x;
            const int tt = idx / DP, i = idx - tt * DP;
            float w = fw[n];
            if (RULE == kBonusMemory) w = i < D ? expm1f(-expf(w + s_w0[i])) : 0.f;
            if (RULE == kChannelDecay) w = i < D ? expm1f(log_sigmoid_f(w + s_w0[i]) * p.inv_tau) : 0.f;
            s_a[buf][tt][i] = RULE == kConstantDecay ? silu_f(fa[n]) : RULE == kChannelDecay ? fa[n] * p.q_scale : fa[n];
            s_k[buf][tt][i] = RULE == kConstantDecay ? silu_f(fk[n]) : fk[n];
            if (RULE != kConstantDecay && RULE != kTokenDecay) s_w[buf][tt][i] = w;
        }
#pragma unroll
        for (int n = 0; n < V_ITEMS; ++n) {
            const int idx = n * THREADS + threadIdx.x;
            if (idx < CHUNK * CTA_COLS) s_v[buf][idx / CTA_COLS][idx % CTA_COLS] = RULE == kConstantDecay ? silu_f(fv[n]) : fv[n];
        }
        if (RULE == 0 && threadIdx.x < CHUNK) s_beta[buf][threadIdx.x] = fb;
        if (RULE == kTokenDecay && threadIdx.x < CHUNK) {
            const float d = softplus_f(fb + dt_bias);
            s_beta[buf][threadIdx.x] = d;
            s_w[buf][threadIdx.x][0] = expm1f(-rate * d);
        }
    };

    fetch(first);
    __syncthreads();            // s_w0 is there
    stash(0);
    __syncthreads();
    int buf = 0;
    for (int c0 = first; c0 < len; c0 += CHUNK, buf ^= 1) {
        const int nt = min(CHUNK, len - c0);
        const bool more = c0 + CHUNK < len;
        if (more) fetch(c0 + CHUNK);
        for (int tt = 0; tt < nt; ++tt) {
            const float4* w4 = reinterpret_cast<const float4*>(&s_w[buf][tt][4 * il]);
            const float4* k4 = reinterpret_cast<const float4*>(&s_k[buf][tt][4 * il]);
            const float4* a4 = reinterpret_cast<const float4*>(&s_a[buf][tt][4 * il]);
            float vj[NC], out[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) vj[c] = s_v[buf][tt][jc + c * COLS];
            // four partial sums a read (fixed order): a single chain of R dependent additions would set the pace
            if (RULE == 0) {
                float d[NC][4], kk[R];
#pragma unroll
                for (int c = 0; c < NC; ++c) d[c][0] = d[c][1] = d[c][2] = d[c][3] = 0.f;
#pragma unroll
                for (int g = 0; g < R / 4; ++g) {
                    const float4 w = w4[LANES * g], k = k4[LANES * g];
                    const float wv[4] = {w.x, w.y, w.z, w.w};
                    kk[4 * g] = k.x; kk[4 * g + 1] = k.y; kk[4 * g + 2] = k.z; kk[4 * g + 3] = k.w;
#pragma unroll
                    for (int c = 0; c < NC; ++c)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            S[c][4 * g + e] = fmaf(S[c][4 * g + e], wv[e], S[c][4 * g + e]);
                            d[c][e] = fmaf(S[c][4 * g + e], kk[4 * g + e], d[c][e]);
                        }
                }
                float u[NC];
#pragma unroll
                for (int c = 0; c < NC; ++c) u[c] = (d[c][0] + d[c][1]) + (d[c][2] + d[c][3]);
#pragma unroll
                for (int o = 1; o < LANES; o <<= 1)
#pragma unroll
                    for (int c = 0; c < NC; ++c) u[c] += __shfl_xor_sync(0xffffffffu, u[c], o);
                const float beta = s_beta[buf][tt];
#pragma unroll
                for (int c = 0; c < NC; ++c) u[c] = beta * (vj[c] - u[c]);
                float acc[NC][4];
#pragma unroll
                for (int c = 0; c < NC; ++c) acc[c][0] = acc[c][1] = acc[c][2] = acc[c][3] = 0.f;
#pragma unroll
                for (int g = 0; g < R / 4; ++g) {
                    const float4 q = a4[LANES * g];
                    const float qv[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                    for (int c = 0; c < NC; ++c)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            S[c][4 * g + e] = fmaf(kk[4 * g + e], u[c], S[c][4 * g + e]);
                            acc[c][e] = fmaf(S[c][4 * g + e], qv[e], acc[c][e]);
                        }
                }
#pragma unroll
                for (int c = 0; c < NC; ++c) out[c] = (acc[c][0] + acc[c][1]) + (acc[c][2] + acc[c][3]);
            } else if (RULE == kChannelDecay || RULE == kConstantDecay || RULE == kTokenDecay) {
                const float plain = RULE == kTokenDecay ? s_w[buf][tt][0] : fade;
                float in[NC];           // what the memory takes of a value
#pragma unroll
                for (int c = 0; c < NC; ++c) in[c] = RULE == kTokenDecay ? s_beta[buf][tt] * vj[c] : vj[c];
                float acc[NC][4];
#pragma unroll
                for (int c = 0; c < NC; ++c) acc[c][0] = acc[c][1] = acc[c][2] = acc[c][3] = 0.f;
#pragma unroll
                for (int g = 0; g < R / 4; ++g) {
                    const float4 k = k4[LANES * g], q = a4[LANES * g];
                    float4 w = make_float4(plain, plain, plain, plain);
                    if (RULE == kChannelDecay) w = w4[LANES * g];
                    const float wv[4] = {w.x, w.y, w.z, w.w}, kv4[4] = {k.x, k.y, k.z, k.w}, qv[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                    for (int c = 0; c < NC; ++c)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            S[c][4 * g + e] = fmaf(kv4[e], in[c], fmaf(wv[e], S[c][4 * g + e], S[c][4 * g + e]));
                            acc[c][e] = fmaf(qv[e], S[c][4 * g + e], acc[c][e]);
                        }
                }
#pragma unroll
                for (int c = 0; c < NC; ++c) out[c] = (acc[c][0] + acc[c][1]) + (acc[c][2] + acc[c][3]);
            } else {
                const float4* b4 = reinterpret_cast<const float4*>(&s_bonus[4 * il]);
                float acc[NC][4];
#pragma unroll
                for (int c = 0; c < NC; ++c) acc[c][0] = acc[c][1] = acc[c][2] = acc[c][3] = 0.f;
#pragma unroll
                for (int g = 0; g < R / 4; ++g) {
                    const float4 w = w4[LANES * g], k = k4[LANES * g], rr = a4[LANES * g], b = b4[LANES * g];
                    const float wv[4] = {w.x, w.y, w.z, w.w}, kv4[4] = {k.x, k.y, k.z, k.w}, rv[4] = {rr.x, rr.y, rr.z, rr.w},
                                bv[4] = {b.x, b.y, b.z, b.w};
                    if (mode == 1) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) decayed[4 * g + e] = fmaf(wv[e], decayed[4 * g + e], decayed[4 * g + e]);
                    }
#pragma unroll
                    for (int c = 0; c < NC; ++c)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const float kv = kv4[e] * vj[c];
                            acc[c][e] = fmaf(rv[e], fmaf(bv[e], kv, S[c][4 * g + e]), acc[c][e]);
                            S[c][4 * g + e] = fmaf(wv[e], S[c][4 * g + e], S[c][4 * g + e]) + kv;
                        }
                }
#pragma unroll
                for (int c = 0; c < NC; ++c) out[c] = (acc[c][0] + acc[c][1]) + (acc[c][2] + acc[c][3]);
            }
#pragma unroll
            for (int o = 1; o < LANES; o <<= 1)
#pragma unroll
                for (int c = 0; c < NC; ++c) out[c] += __shfl_xor_sync(0xffffffffu, out[c], o);
            if (RULE == kTokenDecay) {
#pragma unroll
                for (int c = 0; c < NC; ++c) out[c] = fmaf(skip, vj[c], out[c]);
            }
            if (il == 0 && mode != 1) {
#pragma unroll
                for (int c = 0; c < NC; ++c)
                    if (j0 + c * COLS < DV) p.o[(static_cast<size_t>(start + c0 + tt) * H + h) * DV + j0 + c * COLS] = out[c];
            }
        }
        if (more) stash(buf ^ 1);       // nobody reads that buffer: its chunk was finished before the last barrier
        __syncthreads();
    }
    if (mode != 2) {
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const int i = row_of(r), j = j0 + c * COLS;
                if (i < D && j < DV) S_g[static_cast<size_t>(i) * DV + j] = S[c][r];
            }
    }
    if (mode == 1) {
        if (RULE == 1 && blockIdx.x == 0 && jc == 0) {
#pragma unroll
            for (int r = 0; r < R; ++r)
                if (row_of(r) < D) p.piece_p[(static_cast<size_t>(blockIdx.z) * H + h) * D + row_of(r)] = decayed[r];
        }
        return;
    }
    if (mode == 2 && first != 0) return;          // the CTAs of a request's first piece move the tail
    // The convolution's tail: row m of the new tail is the input of local token len - (taps - 1) + m, which lies in
    // this step or, for a short step, further up in the old tail. Channels are shared out over the CTAs of the request;
    // a channel's rows move in ascending order, so a row is read before it is overwritten.
    if (p.taps > 1) {
        const int keep = p.taps - 1;
        const int all = PIECES ? p.q_len[seq] : len;        // the whole request's tokens, whatever this CTA's piece
        float* tail = p.state + static_cast<size_t>(p.state_slot[seq]) * p.state_stride + p.tail_off;
        const int cta = blockIdx.y * gridDim.x + blockIdx.x, ctas = gridDim.x * gridDim.y;
        for (int c = cta * blockDim.x + threadIdx.x; c < p.C; c += ctas * blockDim.x)
            for (int m = 0; m < keep; ++m) {
                const int src = all - keep + m;
                tail[static_cast<size_t>(m) * p.C + c] = src >= 0 ? load_any(p.proj, static_cast<size_t>(start + src) * p.ld_proj + c, p.proj_bf16)
                                                                 : tail[static_cast<size_t>(m + all) * p.C + c];
            }
    }
}

// Between the two passes over pieces, for a memory whose decay is diagonal: piece_s [z, H, D, DV] holds what every piece
// adds from a zero memory, piece_p [z, H, D] the product of its decays. One thread an entry of S walks the request's pieces
// in order: the memory at a piece's start takes the place of the piece's own sum, and the memory after the last piece goes
// into the state.
static __global__ void __launch_bounds__(256)
pieces_combine_kernel(float* __restrict__ piece_s, const float* __restrict__ piece_p, float* __restrict__ state, long long state_stride,
                      const int32_t* __restrict__ q_len, const int32_t* __restrict__ state_slot, int H, int D, int DV, int piece,
                      int max_pieces) {
    pdl_trigger();
    pdl_wait();
    const int seq = blockIdx.y;
    const int len = q_len[seq];
    if (len <= 0) return;
    const int entry = blockIdx.x * blockDim.x + threadIdx.x;          // over H * D * DV
    if (entry >= H * D * DV) return;
    const int row = entry / DV;                                          // h * D + i
    float* S_g = state + static_cast<size_t>(state_slot[seq]) * state_stride + entry;
    float S = *S_g;
    const int pieces = (len + piece - 1) / piece;
    constexpr int AHEAD = 8;        // pieces whose loads are in flight together
    for (int c0 = 0; c0 < pieces; c0 += AHEAD) {
        float own[AHEAD], decay[AHEAD];
#pragma unroll
        for (int u = 0; u < AHEAD; ++u)
            if (c0 + u < pieces) {
                const size_t z = static_cast<size_t>(seq) * max_pieces + c0 + u;
                own[u] = piece_s[z * H * D * DV + entry];
                decay[u] = piece_p[z * H * D + row];
            }
#pragma unroll
        for (int u = 0; u < AHEAD; ++u)
            if (c0 + u < pieces) {
                piece_s[(static_cast<size_t>(seq) * max_pieces + c0 + u) * H * D * DV + entry] = S;
                S = fmaf(decay[u], S, own[u]);
            }
    }
    *S_g = S;
}

template <int LANES, int R, int CHUNK, int RULE>
int launch_scan_as(const ScanArgs& p, int num_seqs, cudaStream_t stream) {
    constexpr int COLS = kScanThreads / LANES;
    // four columns a thread where the head is wide enough to fill them
    if (p.mode) num_seqs *= p.max_pieces;
    if constexpr (RULE >= kChannelDecay) {      // one chain; long portions of these rules run chunk by chunk (decay_memory.cu)
        if (p.mode) return STRIDE_BAD_ARGUMENT;
        const int cta_cols = p.DV >= 4 * COLS ? 4 * COLS : COLS;
        stride::launch_alone(p.DV >= 4 * COLS ? scan_kernel<LANES, R, 4, CHUNK, RULE, false> : scan_kernel<LANES, R, 1, CHUNK, RULE, false>,
                             dim3((p.DV + cta_cols - 1) / cta_cols, p.H, num_seqs), dim3(kScanThreads), 0, stream, p);
    } else if (p.DV >= 4 * COLS) {
        const dim3 grid((p.DV + 4 * COLS - 1) / (4 * COLS), p.H, num_seqs);
        if (p.mode) stride::launch_alone(scan_kernel<LANES, R, 4, CHUNK, RULE, true>, grid, dim3(kScanThreads), 0, stream, p);
        else stride::launch_alone(scan_kernel<LANES, R, 4, CHUNK, RULE, false>, grid, dim3(kScanThreads), 0, stream, p);
    } else {
        const dim3 grid((p.DV + COLS - 1) / COLS, p.H, num_seqs);
        if (p.mode) stride::launch_alone(scan_kernel<LANES, R, 1, CHUNK, RULE, true>, grid, dim3(kScanThreads), 0, stream, p);
        else stride::launch_alone(scan_kernel<LANES, R, 1, CHUNK, RULE, false>, grid, dim3(kScanThreads), 0, stream, p);
    }
    return STRIDE_LAUNCH_STATUS();
}

template <int RULE>
int launch_scan(const ScanArgs& p, int num_seqs, cudaStream_t stream) {
    if (p.D <= 16) return launch_scan_as<4, 4, 16, RULE>(p, num_seqs, stream);
    if (p.D <= 32) return launch_scan_as<8, 4, 16, RULE>(p, num_seqs, stream);
    if (p.D <= 64) return launch_scan_as<16, 4, 16, RULE>(p, num_seqs, stream);
    if (p.D <= 128) return launch_scan_as<16, 8, 8, RULE>(p, num_seqs, stream);
    if (p.D <= 256) return launch_scan_as<16, 16, 4, RULE>(p, num_seqs, stream);
    return STRIDE_UNSUPPORTED;
}

}  // namespace stride

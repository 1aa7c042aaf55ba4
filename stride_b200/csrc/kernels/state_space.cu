// A selective state space memory with one decay a head and token (Dao and Gu, "Transformers are SSMs: Generalized Models and
// Efficient Algorithms Through Structured State Space Duality"): per head h of group g a matrix S [N, P] in float32 from zero and
// per token
//
//   d = softplus(raw + bias_h);   S <- exp(-exp(a_h) d) S + d B_g x_h^T;   y_h = S^T C_g + skip_h x_h
//
// with x [H, P], B and C [G, N] behind a short causal convolution (with a bias) and SiLU, and behind it a gate and a norm:
//
//   ssm_conv         y_t[c] = silu(b[c] + sum_j w[j, c] u_(t - taps + 1 + j)[c]) for the portions of a step. u is a row of this
//                    step's projection or, before the step's first token, a row of the request's tail.
//   ssm_tail         afterwards: the tails of the portions move on.
//   ssm_scan         one token after the other (memory_scan.cuh): short portions, and the whole 32-bit path, where a token's
//                    output must not depend on how its prompt was cut.
//   ssm_step         a single token of every request (decoding in bfloat16 models): convolution, step size, one pass over S and
//                    the tail's new row in one kernel.
//   ssm_chunks       long portions in bfloat16 models, chunks of 128 tokens side by side on the tensor cores (below).
//   gated_group_norm out = w u / sqrt(mean(u^2) + eps) with u = y silu(z), the mean taken over equal parts of a token's row.
//
// The tail of a request is a ring of `taps` rows: the input of the token at position p lies in row p mod taps. A token reads the
// rows of the taps - 1 positions before it and never the row it writes, so the many CTAs that read a single token's tail need
// not wait for the one that extends it. Rows of positions below zero are never read.
//
// Chunks. With c_i the running sum of the decays' logarithms inside a chunk (c_i <= 0, falling), c_end its last value and S_0 the
// memory before the chunk:
//     y_i   = exp(c_i) S_0^T C_i + sum_(j <= i) (C_i . B_j) exp(c_i - c_j) d_j x_j + skip x_i
//     S_end = exp(c_end) S_0 + sum_j B_j (exp(c_end - c_j) d_j x_j)^T
// No exponent is ever positive. B, C and x are bfloat16 already (they come out of the convolution so), so as operands of
// mma.sync they are exact; what is float32 (S_0, the weighted scores, the weighted x) enters as the sum of two bfloat16
// numbers, which keeps 16 bits of it, with float32 accumulation. Three launches: every chunk's own sum, the memories at the
// chunks' starts (and the tails), the outputs.
#include "memory_scan.cuh"
#include "mma.cuh"

namespace stride {

constexpr int kSsmChunk = 128;          // tokens a chunk
constexpr int kSsmCols = 64;            // columns of S a CTA works on
constexpr int kSsmThreads = 256;
constexpr int kSsmMaxTaps = 16;
constexpr int kSsmMaxState = 256;

// ---------------------------------------------------------------------------------------------------------- convolution
struct SsmConvArgs {
    const void* u;              // [tokens, ld] from the first convolved channel on
    int ld, channels, taps;
    const float* w;             // [taps, channels]
    const float* b;             // [channels]
    const float* ring;          // state rows from the ring on: [taps, channels]
    long long state_stride;
    const int32_t* seq_of_token;
    const int32_t* q_start;
    const int32_t* positions;
    const int32_t* state_slot;
    void* out;                  // [tokens, ld_out]
    int ld_out, tokens;
};

template <typename T, int V>
__device__ __forceinline__ void load_pack(const T* p, float* v) {
    if constexpr (V == 1) {
        v[0] = to_f32(*p);
    } else if constexpr (sizeof(T) == 2) {
        const uint4 r = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            v[2 * i] = f.x;
            v[2 * i + 1] = f.y;
        }
    } else {
#pragma unroll
        for (int i = 0; i < V; i += 4) {
            const float4 r = *reinterpret_cast<const float4*>(p + i);
            v[i] = r.x; v[i + 1] = r.y; v[i + 2] = r.z; v[i + 3] = r.w;
        }
    }
}
template <typename T, int V>
__device__ __forceinline__ void store_pack(T* p, const float* v) {
    if constexpr (V == 1) {
        *p = from_f32<T>(v[0]);
    } else if constexpr (sizeof(T) == 2) {
        uint4 r;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&r);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = r;
    } else {
#pragma unroll
        for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    }
}

// A pack as it lies in memory, to be widened when it is used.
template <typename T, int V>
struct HeldPack {
    float v[V];
    __device__ __forceinline__ void load(const T* p) { load_pack<T, V>(p, v); }
    __device__ __forceinline__ void widen(float* out) const {
#pragma unroll
        for (int e = 0; e < V; ++e) out[e] = v[e];
    }
};
template <>
struct HeldPack<__nv_bfloat16, 8> {
    uint4 raw;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { raw = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void widen(float* out) const { load_pack<__nv_bfloat16, 8>(reinterpret_cast<const __nv_bfloat16*>(&raw), out); }
};

// SiLU for an output of type T: what is rounded to 16 bits takes the quick form.
template <typename T>
__device__ __forceinline__ float silu_for(float z) { return sizeof(T) == 2 ? silu_quick(z) : silu_f(z); }

// A thread: V neighbouring channels of `run` consecutive rows. TAPS > 0: that many taps, the last inputs kept in registers from
// row to row, four rows asked for at a time; TAPS 0: any number, every input read again.
template <typename TI, typename TO, int V, int TAPS>
__global__ void __launch_bounds__(128, 5)
ssm_conv_kernel(const SsmConvArgs p, int run) {
    pdl_trigger();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (c >= p.channels) return;
    const int taps = TAPS > 0 ? TAPS : p.taps;
    constexpr int HELD = TAPS > 0 ? TAPS : 1;
    float w[HELD][V], bias[V];
    if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < HELD; ++j) load_pack<float, V>(p.w + static_cast<size_t>(j) * p.channels + c, w[j]);
    }
    load_pack<float, V>(p.b + c, bias);
    pdl_wait();
    const TI* u = static_cast<const TI*>(p.u) + c;
    TO* out = static_cast<TO*>(p.out) + c;
    // the input `back` tokens before local token `local` (back >= 1) of a request
    auto earlier = [&](int start, int local, int at, int slot, int back, float* v) {
        if (local - back >= 0) {
            load_pack<TI, V>(u + static_cast<size_t>(start + local - back) * p.ld, v);
        } else if (at - back >= 0) {
            load_pack<float, V>(p.ring + static_cast<size_t>(slot) * p.state_stride + static_cast<size_t>((at - back) % taps) * p.channels + c, v);
        } else {
#pragma unroll
            for (int e = 0; e < V; ++e) v[e] = 0.f;
        }
    };
    float hist[HELD][V];            // inputs of tokens t - TAPS + 1 .. t (the last slot: t)
    int held_seq = -1;
    const int t0 = blockIdx.y * run, t1 = min(t0 + run, p.tokens);
    constexpr int ROWS = 4;
    for (int tb = t0; tb < t1; tb += ROWS) {
        HeldPack<TI, V> fresh[ROWS];
        int seqs[ROWS];
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            seqs[r] = -1;
            if (tb + r < t1) {
                seqs[r] = p.seq_of_token[tb + r];
                fresh[r].load(u + static_cast<size_t>(tb + r) * p.ld);
            }
        }
#pragma unroll
        for (int r = 0; r < ROWS; ++r) {
            const int t = tb + r, seq = seqs[r];
            if (seq < 0) {
                held_seq = -1;
                continue;
            }
            float y[V];
#pragma unroll
            for (int e = 0; e < V; ++e) y[e] = bias[e];
            if (TAPS > 0) {
                if (seq == held_seq) {
#pragma unroll
                    for (int j = 0; j + 1 < HELD; ++j)
#pragma unroll
                        for (int e = 0; e < V; ++e) hist[j][e] = hist[j + 1][e];
                } else {
                    const int start = p.q_start[seq], slot = p.state_slot[seq], at = p.positions[t];
#pragma unroll
                    for (int j = 0; j + 1 < HELD; ++j) earlier(start, t - start, at, slot, HELD - 1 - j, hist[j]);
                    held_seq = seq;
                }
                fresh[r].widen(hist[HELD - 1]);
#pragma unroll
                for (int j = 0; j < HELD; ++j)
#pragma unroll
                    for (int e = 0; e < V; ++e) y[e] = fmaf(w[j][e], hist[j][e], y[e]);
            } else {
                const int start = p.q_start[seq], slot = p.state_slot[seq], at = p.positions[t];
                for (int j = 0; j < taps; ++j) {
                    float v[V], f[V];
                    load_pack<float, V>(p.w + static_cast<size_t>(j) * p.channels + c, f);
                    if (j + 1 < taps) earlier(start, t - start, at, slot, taps - 1 - j, v);
                    else fresh[r].widen(v);
#pragma unroll
                    for (int e = 0; e < V; ++e) y[e] = fmaf(f[e], v[e], y[e]);
                }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) y[e] = silu_for<TO>(y[e]);
            store_pack<TO, V>(out + static_cast<size_t>(t) * p.ld_out, y);
        }
    }
}

struct SsmTailArgs {
    const void* u;
    int ld, u_bf16, channels, taps;
    float* ring;
    long long state_stride;
    const int32_t* q_start;
    const int32_t* q_len;
    const int32_t* positions;
    const int32_t* state_slot;
};

// The rows of the ring that the request's last min(len, taps - 1) tokens of this step own.
__device__ __forceinline__ void move_tail(const SsmTailArgs& p, int seq, int c) {
    const int len = p.q_len[seq], start = p.q_start[seq], first = p.positions[start];
    float* ring = p.ring + static_cast<size_t>(p.state_slot[seq]) * p.state_stride;
    for (int i = max(0, len - (p.taps - 1)); i < len; ++i)
        ring[static_cast<size_t>((first + i) % p.taps) * p.channels + c] = load_any(p.u, static_cast<size_t>(start + i) * p.ld + c, p.u_bf16);
}

static __global__ void __launch_bounds__(128)
ssm_tail_kernel(const SsmTailArgs p) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= p.channels || p.q_len[blockIdx.y] <= 0) return;
    move_tail(p, blockIdx.y, c);
}

// ------------------------------------------------------------------------------------------------------------ one token
struct SsmStepArgs {
    const void* u;              // [tokens, ld] from the first convolved channel on: x [H, P], B [G, N], C [G, N]
    int ld, u_bf16;
    const float* raw;           // [tokens, ld_raw]: step sizes before bias and softplus
    int ld_raw;
    const float* w;
    const float* b;
    const float* dt_bias;
    const float* a_log;
    const float* skip;
    float* y;                   // [tokens, H * P]
    float* state;               // S of head h at h * N * P; the ring at ring_off
    long long state_stride, ring_off;
    const int32_t* q_start;
    const int32_t* q_len;
    const int32_t* positions;
    const int32_t* state_slot;
    int H, G, N, P, taps;
};

// Grid (tiles of COLS columns, heads, requests). A row of a tile is COLS / 4 lanes of 16 bytes; the rows of S are spread over the
// rest of the CTA, whose shares of S^T C meet in shared memory.
template <int COLS>
__global__ void __launch_bounds__(kSsmThreads)
ssm_step_kernel(const SsmStepArgs p) {
    constexpr int ROW_LANES = COLS / 4, ROWS = kSsmThreads / ROW_LANES;
    __shared__ float s_x[COLS], s_b[kSsmMaxState], s_c[kSsmMaxState];
    __shared__ __align__(16) float red[ROWS][COLS];
    pdl_trigger();
    const int seq = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * COLS;
    const int N = p.N, P = p.P, g = h / (p.H / p.G);
    const int lane = threadIdx.x % ROW_LANES, row = threadIdx.x / ROW_LANES;
    const bool live = col0 + 4 * lane < P;
    const float rate = expf(p.a_log[h]), dt_bias = p.dt_bias[h], skip = p.skip[h];
    pdl_wait();
    if (p.q_len[seq] <= 0) return;
    float* mine = p.state + static_cast<size_t>(p.state_slot[seq]) * p.state_stride;
    float* S_g = mine + static_cast<size_t>(h) * N * P + col0 + 4 * lane;
    constexpr int AHEAD = 8;
    float4 S[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k)
        if (live && row + ROWS * k < N) S[k] = *reinterpret_cast<const float4*>(S_g + static_cast<size_t>(row + ROWS * k) * P);
    const size_t t = static_cast<size_t>(p.q_start[seq]);
    const int at = p.positions[t], C = p.H * P + 2 * p.G * N;
    float* ring = mine + p.ring_off;
    for (int i = threadIdx.x; i < COLS + 2 * N; i += kSsmThreads) {
        // x of this tile, then the group's B, then its C
        int c = -1;
        if (i < COLS) {
            if (col0 + i < P) c = h * P + col0 + i;
        } else if (i < COLS + N) {
            c = p.H * P + g * N + i - COLS;
        } else {
            c = p.H * P + p.G * N + g * N + i - COLS - N;
        }
        float v = 0.f;
        if (c >= 0) {
            const float now = load_any(p.u, t * p.ld + c, p.u_bf16), last = p.w[static_cast<size_t>(p.taps - 1) * C + c];
            v = p.b[c];
            for (int j0 = 0; j0 + 1 < p.taps; j0 += 3) {        // three earlier inputs are asked for together
                float was[3], f[3];
#pragma unroll
                for (int e = 0; e < 3; ++e) {
                    const int back = p.taps - 1 - j0 - e;
                    was[e] = f[e] = 0.f;
                    if (back > 0 && at >= back) {
                        was[e] = ring[static_cast<size_t>((at - back) % p.taps) * C + c];
                        f[e] = p.w[static_cast<size_t>(j0 + e) * C + c];
                    }
                }
#pragma unroll
                for (int e = 0; e < 3; ++e) v = fmaf(f[e], was[e], v);
            }
            v = silu_f(fmaf(last, now, v));
            // one writer a channel: x the CTA whose columns they are, B and C the first CTA of the group
            if (p.taps > 1 && (i < COLS || (blockIdx.x == 0 && h == g * (p.H / p.G)))) ring[static_cast<size_t>(at % p.taps) * C + c] = now;
        }
        if (i < COLS) s_x[i] = v;
        else if (i < COLS + N) s_b[i - COLS] = v;
        else s_c[i - COLS - N] = v;
    }
    const float d = softplus_f(p.raw[t * p.ld_raw + h] + dt_bias), keep = expm1f(-rate * d);
    __syncthreads();
    float in[4], acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int e = 0; e < 4; ++e) in[e] = d * s_x[4 * lane + e];
    for (int n0 = 0; n0 < N; n0 += ROWS * AHEAD) {
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            const int n = n0 + row + ROWS * k;
            if (live && n < N) {
                const float b = s_b[n], q = s_c[n];
                float x[4] = {S[k].x, S[k].y, S[k].z, S[k].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    x[e] = fmaf(b, in[e], fmaf(keep, x[e], x[e]));
                    acc[e] = fmaf(q, x[e], acc[e]);
                }
                *reinterpret_cast<float4*>(S_g + static_cast<size_t>(n) * P) = make_float4(x[0], x[1], x[2], x[3]);
            }
        }
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            const int n = n0 + ROWS * AHEAD + row + ROWS * k;
            if (live && n < N) S[k] = *reinterpret_cast<const float4*>(S_g + static_cast<size_t>(n) * P);
        }
    }
    *reinterpret_cast<float4*>(&red[row][4 * lane]) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    __syncthreads();
    if (threadIdx.x < COLS && col0 + threadIdx.x < P) {
        float sum = 0.f;
#pragma unroll
        for (int r = 0; r < ROWS; ++r) sum += red[r][threadIdx.x];
        p.y[(t * p.H + h) * P + col0 + threadIdx.x] = fmaf(skip, s_x[threadIdx.x], sum);
    }
}

// --------------------------------------------------------------------------------------------------------------- chunks
struct SsmChunkArgs {
    const __nv_bfloat16* x;     // [tokens, ld], head h at column h * P
    const __nv_bfloat16* B;     // group g at column g * N
    const __nv_bfloat16* C;
    int ld;
    const float* raw;           // [tokens, ld_raw]
    int ld_raw;
    const float* dt_bias;
    const float* a_log;
    const float* skip;
    float* y;                   // [tokens, H * P]
    float* piece_s;             // [seqs * max_pieces, H, N, P]: a chunk's own sum, then the memory at its start
    float* piece_p;             // [seqs * max_pieces, H]: exp(c_end)
    const int32_t* q_start;
    const int32_t* q_len;
    int H, G, N, P, max_pieces;
    int vec;                    // rows of B, C and x can be read in packs of 8
};

// The raw step sizes of a chunk's tokens, four neighbouring tokens a lane of the first warp; then their d_j and the running sums c_j.
__device__ __forceinline__ void chunk_raw(const SsmChunkArgs& p, int h, size_t row0, int nt, float (&raw)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const int j = 4 * threadIdx.x + e;
        raw[e] = threadIdx.x < 32 && j < nt ? p.raw[(row0 + j) * p.ld_raw + h] : 0.f;
    }
}
__device__ __forceinline__ void chunk_decays(const SsmChunkArgs& p, int h, int nt, const float (&raw)[4], float* s_d, float* s_c) {
    if (threadIdx.x >= 32) return;
    const float rate = expf(p.a_log[h]), bias = p.dt_bias[h];
    const int lane = threadIdx.x;
    float d[4], c[4], sum = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        d[e] = 4 * lane + e < nt ? softplus_f(raw[e] + bias) : 0.f;
        sum -= rate * d[e];
        c[e] = sum;
    }
    float before = sum;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float v = __shfl_up_sync(0xffffffffu, before, o);
        if (lane >= o) before += v;
    }
    before = __shfl_up_sync(0xffffffffu, before, 1);
    if (lane == 0) before = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        s_d[4 * lane + e] = d[e];
        s_c[4 * lane + e] = before + c[e];
    }
}

// [rows][cols] bfloat16 of global rows (stride ld) into shared memory (stride LDS), zeros beyond nt rows and `width` columns.
template <int ROWS, int COLS, int LDS>
__device__ __forceinline__ void stage_bf16(__nv_bfloat16* dst, const __nv_bfloat16* src, int ld, int nt, int width, bool vec) {
    if (vec) {
        constexpr int PACKS = ROWS * COLS / 8;
#pragma unroll 8
        for (int idx = threadIdx.x; idx < PACKS; idx += kSsmThreads) {
            const int r = idx / (COLS / 8), c = (idx % (COLS / 8)) * 8;
            const uint4 v = r < nt && c < width ? *reinterpret_cast<const uint4*>(src + static_cast<size_t>(r) * ld + c) : make_uint4(0, 0, 0, 0);
            *reinterpret_cast<uint4*>(dst + r * LDS + c) = v;
        }
        return;
    }
    for (int idx = threadIdx.x; idx < ROWS * COLS; idx += kSsmThreads) {
        const int r = idx / COLS, c = idx % COLS;
        dst[r * LDS + c] = r < nt && c < width ? src[static_cast<size_t>(r) * ld + c] : __float2bfloat16_rn(0.f);
    }
}

// The same by asynchronous copies where rows allow them (cp_async_wait and a barrier before the tile is read).
template <int ROWS, int COLS, int LDS>
__device__ __forceinline__ void stage_async(__nv_bfloat16* dst, const __nv_bfloat16* src, int ld, int nt, int width, bool vec) {
    if (!vec) return stage_bf16<ROWS, COLS, LDS>(dst, src, ld, nt, width, false);
#pragma unroll
    for (int n = 0; n < ROWS * COLS / 8 / kSsmThreads; ++n) {
        const int idx = n * kSsmThreads + threadIdx.x, r = idx / (COLS / 8), c = (idx % (COLS / 8)) * 8;
        if (r < nt && c < width) cp_async_16(dst + r * LDS + c, src + static_cast<size_t>(r) * ld + c);
        else *reinterpret_cast<uint4*>(dst + r * LDS + c) = make_uint4(0, 0, 0, 0);
    }
}

// v as the sum of two bfloat16 numbers.
__device__ __forceinline__ void split_bf16(float v, __nv_bfloat16& hi, __nv_bfloat16& lo) {
    hi = __float2bfloat16_rn(v);
    lo = __float2bfloat16_rn(v - __bfloat162float(hi));
}
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
    __nv_bfloat162 h, l;
    split_bf16(a, h.x, l.x);
    split_bf16(b, h.y, l.y);
    hi = *reinterpret_cast<uint32_t*>(&h);
    lo = *reinterpret_cast<uint32_t*>(&l);
}

constexpr int kLdX = kSsmCols + 8;              // row strides in shared memory: 16-byte rows that fall into different banks
template <int NP>
__host__ __device__ constexpr int ld_n() { return NP + 8; }

template <int NP>
constexpr int sum_smem_bytes() { return (kSsmChunk * ld_n<NP>() + 2 * kSsmChunk * kLdX) * 2; }
template <int NP>
constexpr int out_smem_bytes() { return (kSsmChunk * ld_n<NP>() + kSsmChunk * kLdX + 2 * NP * kLdX) * 2; }

// piece_s[z, h] = sum_j B_j (exp(c_end - c_j) d_j x_j)^T, piece_p[z, h] = exp(c_end). NP: N padded. Grid (column tiles, heads, chunks).
template <int NP>
__global__ void __launch_bounds__(kSsmThreads)
ssm_chunk_sum_kernel(const SsmChunkArgs p) {
    constexpr int LDN = ld_n<NP>();
    extern __shared__ __align__(16) unsigned char raw_smem[];
    __nv_bfloat16* Bs = reinterpret_cast<__nv_bfloat16*>(raw_smem);     // [kSsmChunk][LDN]
    __nv_bfloat16* xh = Bs + kSsmChunk * LDN;                           // [kSsmChunk][kLdX]: high parts of the weighted x
    __nv_bfloat16* xl = xh + kSsmChunk * kLdX;                          // low parts
    __shared__ float s_d[kSsmChunk], s_c[kSsmChunk];
    pdl_trigger();
    const int z = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * kSsmCols;
    const int seq = z / p.max_pieces, first = (z % p.max_pieces) * kSsmChunk;
    const int nt = min(p.q_len[seq] - first, kSsmChunk);
    if (nt <= 0) return;
    pdl_wait();
    const int N = p.N, P = p.P, g = h / (p.H / p.G);
    const size_t row0 = static_cast<size_t>(p.q_start[seq] + first);
    const __nv_bfloat16* x = p.x + row0 * p.ld + h * P + col0;
    const int width = min(P - col0, kSsmCols);
    // everything the CTA reads is asked for before anything is waited for
    float raw[4];
    chunk_raw(p, h, row0, nt, raw);
    constexpr int PACKS = kSsmChunk * kSsmCols / 8 / kSsmThreads;
    uint4 rx[PACKS];
    if (p.vec) {
#pragma unroll
        for (int n = 0; n < PACKS; ++n) {
            const int idx = n * kSsmThreads + threadIdx.x, j = idx / (kSsmCols / 8), c = (idx % (kSsmCols / 8)) * 8;
            rx[n] = j < nt && c < width ? *reinterpret_cast<const uint4*>(x + static_cast<size_t>(j) * p.ld + c) : make_uint4(0, 0, 0, 0);
        }
    }
    stage_async<kSsmChunk, NP, LDN>(Bs, p.B + row0 * p.ld + g * N, p.ld, nt, N, p.vec);
    cp_async_commit();
    chunk_decays(p, h, nt, raw, s_d, s_c);
    __syncthreads();
    const float end = s_c[nt - 1];
    if (p.vec) {
#pragma unroll
        for (int n = 0; n < PACKS; ++n) {
            const int idx = n * kSsmThreads + threadIdx.x, j = idx / (kSsmCols / 8), c = (idx % (kSsmCols / 8)) * 8;
            const float f = expf(end - s_c[j]) * s_d[j];
            const __nv_bfloat162* v = reinterpret_cast<const __nv_bfloat162*>(&rx[n]);
            uint4 hi, lo;
            uint32_t* ph = reinterpret_cast<uint32_t*>(&hi);
            uint32_t* pl = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 q = __bfloat1622float2(v[e]);
                split_pair(q.x * f, q.y * f, ph[e], pl[e]);
            }
            *reinterpret_cast<uint4*>(xh + j * kLdX + c) = hi;
            *reinterpret_cast<uint4*>(xl + j * kLdX + c) = lo;
        }
    } else {
        for (int idx = threadIdx.x; idx < kSsmChunk * kSsmCols; idx += kSsmThreads) {
            const int j = idx / kSsmCols, c = idx % kSsmCols;
            const float v = j < nt && c < width ? __bfloat162float(x[static_cast<size_t>(j) * p.ld + c]) * expf(end - s_c[j]) * s_d[j] : 0.f;
            split_bf16(v, xh[j * kLdX + c], xl[j * kLdX + c]);
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    if (blockIdx.x == 0 && threadIdx.x == 0) p.piece_p[static_cast<size_t>(z) * p.H + h] = expf(end);
    // warps over row tiles of 16 first, over columns with what is left
    constexpr int TILES = NP / 16, MW = TILES < 8 ? TILES : 8, CW = 8 / MW, MT = TILES / MW, NT = kSsmCols / CW / 8;
    static_assert(NT % 2 == 0, "column tiles are read in pairs");
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wm = warp % MW, wc = warp / MW;
    float acc[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < NT; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.f;
    const int steps = (nt + 15) / 16;
    for (int k = 0; k < steps; ++k) {
        uint32_t a[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) {      // A = B^T: rows are state channels, stored token by token
            const int r = k * 16 + (lane & 7) + ((lane >> 4) << 3), c = (wm * MT + m) * 16 + (((lane >> 3) & 1) << 3);
            ldmatrix_x4_trans(a[m], smem_addr(Bs + r * LDN + c));
        }
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
            const int r = k * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), c = wc * NT * 8 + n * 8 + ((lane >> 4) << 3);
            uint32_t bh[4], bl[4];
            ldmatrix_x4_trans(bh, smem_addr(xh + r * kLdX + c));
            ldmatrix_x4_trans(bl, smem_addr(xl + r * kLdX + c));
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                mma_bf16_16816(acc[m][n], a[m], bh[0], bh[1]);
                mma_bf16_16816(acc[m][n], a[m], bl[0], bl[1]);
                mma_bf16_16816(acc[m][n + 1], a[m], bh[2], bh[3]);
                mma_bf16_16816(acc[m][n + 1], a[m], bl[2], bl[3]);
            }
        }
    }
    float* out = p.piece_s + (static_cast<size_t>(z) * p.H + h) * N * P;
    const bool even = P % 2 == 0;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int r = (wm * MT + m) * 16 + (lane >> 2) + 8 * half, c = col0 + wc * NT * 8 + n * 8 + 2 * (lane & 3);
                if (r >= N || c >= P) continue;
                float* dst = out + static_cast<size_t>(r) * P + c;
                if (even) {
                    *reinterpret_cast<float2*>(dst) = make_float2(acc[m][n][2 * half], acc[m][n][2 * half + 1]);
                } else {
                    dst[0] = acc[m][n][2 * half];
                    if (c + 1 < P) dst[1] = acc[m][n][2 * half + 1];
                }
            }
}

// Between the two: piece_s becomes the memory at every chunk's start, the state the memory after the last one. V neighbouring
// entries a thread. The blocks behind the entries' move the tails.
template <int V>
__global__ void __launch_bounds__(256)
ssm_combine_kernel(const SsmChunkArgs p, float* __restrict__ state, long long state_stride, const int32_t* __restrict__ state_slot,
                   int entry_blocks, const SsmTailArgs tail) {
    pdl_trigger();
    const int seq = blockIdx.y, len = p.q_len[seq];
    if (len <= 0) return;
    if (static_cast<int>(blockIdx.x) >= entry_blocks) {
        const int c = (blockIdx.x - entry_blocks) * blockDim.x + threadIdx.x;
        if (c >= tail.channels) return;
        pdl_wait();
        move_tail(tail, seq, c);
        return;
    }
    const long long NPH = static_cast<long long>(p.H) * p.N * p.P, entry = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) * V;
    if (entry >= NPH) return;
    pdl_wait();
    const int h = static_cast<int>(entry / (static_cast<long long>(p.N) * p.P));
    float* S_g = state + static_cast<size_t>(state_slot[seq]) * state_stride + entry;
    float S[V];
    load_pack<float, V>(S_g, S);
    const int pieces = (len + kSsmChunk - 1) / kSsmChunk;
    constexpr int AHEAD = 8;
    for (int c0 = 0; c0 < pieces; c0 += AHEAD) {
        float own[AHEAD][V], decay[AHEAD];
#pragma unroll
        for (int k = 0; k < AHEAD; ++k)
            if (c0 + k < pieces) {
                const size_t z = static_cast<size_t>(seq) * p.max_pieces + c0 + k;
                load_pack<float, V>(p.piece_s + z * NPH + entry, own[k]);
                decay[k] = p.piece_p[z * p.H + h];
            }
#pragma unroll
        for (int k = 0; k < AHEAD; ++k)
            if (c0 + k < pieces) {
                store_pack<float, V>(p.piece_s + (static_cast<size_t>(seq) * p.max_pieces + c0 + k) * NPH + entry, S);
#pragma unroll
                for (int e = 0; e < V; ++e) S[e] = fmaf(decay[k], S[e], own[k][e]);
            }
    }
    store_pack<float, V>(S_g, S);
}

// Outputs of a chunk from the memory at its start (piece_s by now). A warp: 16 tokens, all columns of the tile.
template <int NP>
__global__ void __launch_bounds__(kSsmThreads)
ssm_chunk_out_kernel(const SsmChunkArgs p) {
    constexpr int LDN = ld_n<NP>(), NT = kSsmCols / 8;
    extern __shared__ __align__(16) unsigned char raw_smem[];
    __nv_bfloat16* BCs = reinterpret_cast<__nv_bfloat16*>(raw_smem);    // [kSsmChunk][LDN]: C, then B
    __nv_bfloat16* xs = BCs + kSsmChunk * LDN;                          // [kSsmChunk][kLdX]
    __nv_bfloat16* Sh = xs + kSsmChunk * kLdX;                          // [NP][kLdX]: high parts of the memory
    __nv_bfloat16* Sl = Sh + NP * kLdX;                                 // low parts
    __shared__ float s_d[kSsmChunk], s_c[kSsmChunk];
    pdl_trigger();
    const int z = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * kSsmCols;
    const int seq = z / p.max_pieces, first = (z % p.max_pieces) * kSsmChunk;
    const int nt = min(p.q_len[seq] - first, kSsmChunk);
    if (nt <= 0) return;
    pdl_wait();
    const int N = p.N, P = p.P, g = h / (p.H / p.G);
    const size_t row0 = static_cast<size_t>(p.q_start[seq] + first);
    const int width = min(P - col0, kSsmCols);
    // everything the CTA reads is asked for before anything is waited for: C and x go to shared memory by asynchronous copies, S
    // (of up to 128 rows) and B, whose place C holds at first, to registers
    float raw[4];
    chunk_raw(p, h, row0, nt, raw);
    stage_async<kSsmChunk, NP, LDN>(BCs, p.C + row0 * p.ld + g * N, p.ld, nt, N, p.vec);
    stage_async<kSsmChunk, kSsmCols, kLdX>(xs, p.x + row0 * p.ld + h * P + col0, p.ld, nt, width, p.vec);
    cp_async_commit();
    constexpr bool HELD = NP <= 128;
    constexpr int B_PACKS = HELD ? kSsmChunk * NP / 8 / kSsmThreads : 1;
    const __nv_bfloat16* B = p.B + row0 * p.ld + g * N;
    uint4 rb[B_PACKS];
    if (HELD && p.vec) {
#pragma unroll
        for (int n = 0; n < B_PACKS; ++n) {
            const int idx = n * kSsmThreads + threadIdx.x, r = idx / (NP / 8), c = (idx % (NP / 8)) * 8;
            rb[n] = r < nt && c < N ? *reinterpret_cast<const uint4*>(B + static_cast<size_t>(r) * p.ld + c) : make_uint4(0, 0, 0, 0);
        }
    }
    const float* S = p.piece_s + (static_cast<size_t>(z) * p.H + h) * N * P + col0;
    chunk_decays(p, h, nt, raw, s_d, s_c);
    if (P % 4 == 0) {
        constexpr int S_PACKS = NP * kSsmCols / 4 / kSsmThreads;        // 16 bytes each
        constexpr int TURN = S_PACKS < 8 ? S_PACKS : 8;
#pragma unroll
        for (int n0 = 0; n0 < S_PACKS; n0 += TURN) {
            float4 rs[TURN];
#pragma unroll
            for (int n = 0; n < TURN; ++n) {
                const int idx = (n0 + n) * kSsmThreads + threadIdx.x, r = idx / (kSsmCols / 4), c = (idx % (kSsmCols / 4)) * 4;
                rs[n] = r < N && c < width ? *reinterpret_cast<const float4*>(S + static_cast<size_t>(r) * P + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int n = 0; n < TURN; ++n) {
                const int idx = (n0 + n) * kSsmThreads + threadIdx.x, r = idx / (kSsmCols / 4), c = (idx % (kSsmCols / 4)) * 4;
                uint2 hi, lo;
                split_pair(rs[n].x, rs[n].y, hi.x, lo.x);
                split_pair(rs[n].z, rs[n].w, hi.y, lo.y);
                *reinterpret_cast<uint2*>(Sh + r * kLdX + c) = hi;
                *reinterpret_cast<uint2*>(Sl + r * kLdX + c) = lo;
            }
        }
    } else {
        for (int idx = threadIdx.x; idx < NP * kSsmCols; idx += kSsmThreads) {
            const int r = idx / kSsmCols, c = idx % kSsmCols;
            split_bf16(r < N && c < width ? S[static_cast<size_t>(r) * P + c] : 0.f, Sh[r * kLdX + c], Sl[r * kLdX + c]);
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, i0 = warp * 16;
    const bool busy = i0 < nt;                  // the warp has tokens
    uint32_t cf[NP / 16][4];                    // this warp's rows of C, for both products
#pragma unroll
    for (int k = 0; k < NP / 16; ++k) ldmatrix_x4(cf[k], smem_addr(BCs + (i0 + (lane & 15)) * LDN + k * 16 + ((lane >> 4) << 3)));
    __syncthreads();
    if (HELD && p.vec) {
#pragma unroll
        for (int n = 0; n < B_PACKS; ++n) {
            const int idx = n * kSsmThreads + threadIdx.x, r = idx / (NP / 8), c = (idx % (NP / 8)) * 8;
            *reinterpret_cast<uint4*>(BCs + r * LDN + c) = rb[n];
        }
    } else {
        stage_bf16<kSsmChunk, NP, LDN>(BCs, B, p.ld, nt, N, p.vec);
    }
    float acc[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
    if (busy) {
#pragma unroll
        for (int k = 0; k < NP / 16; ++k)
#pragma unroll
            for (int n = 0; n < NT; n += 2) {
                const int r = k * 16 + (lane & 7) + (((lane >> 3) & 1) << 3), c = n * 8 + ((lane >> 4) << 3);
                uint32_t bh[4], bl[4];
                ldmatrix_x4_trans(bh, smem_addr(Sh + r * kLdX + c));
                ldmatrix_x4_trans(bl, smem_addr(Sl + r * kLdX + c));
                mma_bf16_16816(acc[n], cf[k], bh[0], bh[1]);
                mma_bf16_16816(acc[n], cf[k], bl[0], bl[1]);
                mma_bf16_16816(acc[n + 1], cf[k], bh[2], bh[3]);
                mma_bf16_16816(acc[n + 1], cf[k], bl[2], bl[3]);
            }
    }
    const int ia = i0 + (lane >> 2), ib = ia + 8;       // the two tokens of this lane
    const float ca = s_c[ia], cb = s_c[ib], ea = expf(ca), eb = expf(cb);
#pragma unroll
    for (int n = 0; n < NT; ++n) {
        acc[n][0] *= ea;
        acc[n][1] *= ea;
        acc[n][2] *= eb;
        acc[n][3] *= eb;
    }
    __syncthreads();
    if (!busy) return;
    for (int j0 = 0; j0 <= i0; j0 += 16) {
        float s[2][4] = {};
#pragma unroll
        for (int k = 0; k < NP / 16; ++k) {
            uint32_t b[4];
            ldmatrix_x4(b, smem_addr(BCs + (j0 + (lane & 7) + ((lane >> 4) << 3)) * LDN + k * 16 + (((lane >> 3) & 1) << 3)));
            mma_bf16_16816(s[0], cf[k], b[0], b[1]);
            mma_bf16_16816(s[1], cf[k], b[2], b[3]);
        }
#pragma unroll
        for (int q = 0; q < 2; ++q)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int j = j0 + 8 * q + 2 * (lane & 3) + e;
                const float cj = s_c[j], dj = s_d[j];
                s[q][e] = j <= ia ? s[q][e] * __expf(ca - cj) * dj : 0.f;
                s[q][2 + e] = j <= ib ? s[q][2 + e] * __expf(cb - cj) * dj : 0.f;
            }
        uint32_t ah[4], al[4];
        split_pair(s[0][0], s[0][1], ah[0], al[0]);
        split_pair(s[0][2], s[0][3], ah[1], al[1]);
        split_pair(s[1][0], s[1][1], ah[2], al[2]);
        split_pair(s[1][2], s[1][3], ah[3], al[3]);
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
            const int r = j0 + (lane & 7) + (((lane >> 3) & 1) << 3), c = n * 8 + ((lane >> 4) << 3);
            uint32_t b[4];
            ldmatrix_x4_trans(b, smem_addr(xs + r * kLdX + c));
            mma_bf16_16816(acc[n], ah, b[0], b[1]);
            mma_bf16_16816(acc[n], al, b[0], b[1]);
            mma_bf16_16816(acc[n + 1], ah, b[2], b[3]);
            mma_bf16_16816(acc[n + 1], al, b[2], b[3]);
        }
    }
    const float skip = p.skip[h];
    const bool even = P % 2 == 0;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int i = half ? ib : ia, c = n * 8 + 2 * (lane & 3);
            if (i >= nt || c >= width) continue;
            const float v0 = fmaf(skip, __bfloat162float(xs[i * kLdX + c]), acc[n][2 * half]);
            const float v1 = fmaf(skip, __bfloat162float(xs[i * kLdX + c + 1]), acc[n][2 * half + 1]);
            float* dst = p.y + ((row0 + i) * p.H + h) * P + col0 + c;
            if (even) {
                *reinterpret_cast<float2*>(dst) = make_float2(v0, v1);
            } else {
                dst[0] = v0;
                if (c + 1 < width) dst[1] = v1;
            }
        }
}

template <int NP>
int launch_ssm_chunks(const SsmChunkArgs& p, float* state, long long state_stride, const int32_t* state_slot, int num_seqs, const SsmTailArgs& tail,
                      cudaStream_t stream) {
    const dim3 grid((p.P + kSsmCols - 1) / kSsmCols, p.H, num_seqs * p.max_pieces), block(kSsmThreads);
    cudaError_t e = cudaFuncSetAttribute(ssm_chunk_sum_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, sum_smem_bytes<NP>());
    if (e == cudaSuccess) e = cudaFuncSetAttribute(ssm_chunk_out_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, out_smem_bytes<NP>());
    if (e != cudaSuccess) return static_cast<int>(e);
    stride::launch(ssm_chunk_sum_kernel<NP>, grid, block, sum_smem_bytes<NP>(), stream, p);
    const bool packs = (p.N * p.P) % 4 == 0 && state_stride % 4 == 0 && reinterpret_cast<uintptr_t>(state) % 16 == 0;
    const long long entries = static_cast<long long>(p.H) * p.N * p.P, threads = packs ? entries / 4 : entries;
    const int entry_blocks = static_cast<int>((threads + 255) / 256), tail_blocks = tail.taps > 1 ? (tail.channels + 255) / 256 : 0;
    stride::launch(packs ? ssm_combine_kernel<4> : ssm_combine_kernel<1>, dim3(entry_blocks + tail_blocks, num_seqs), dim3(256), 0, stream, p, state,
                   state_stride, state_slot, entry_blocks, tail);
    stride::launch(ssm_chunk_out_kernel<NP>, grid, block, out_smem_bytes<NP>(), stream, p);
    return STRIDE_LAUNCH_STATUS();
}

// ---------------------------------------------------------------------------------------------------- gate, then norm
// One group of THREADS threads a (token, part); V columns a thread and turn. z: the gate's logits in TZ.
template <typename TZ, typename TO, int THREADS, int V>
__global__ void __launch_bounds__(256)
gated_group_norm_kernel(const float* __restrict__ y, const TZ* __restrict__ z, int ld_z, const float* __restrict__ weight, TO* __restrict__ out,
                        int width, int parts, long long pairs, float eps) {
    constexpr int HELD = 8;             // turns whose values stay in registers; later ones are worked out twice
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const long long pair = THREADS == 32 ? static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5) : blockIdx.x;
    if (pair >= pairs) return;          // whole warps leave, and only where a warp is the group
    const int me = threadIdx.x % THREADS, part = static_cast<int>(pair % parts);
    const size_t t = static_cast<size_t>(pair / parts);
    const float* row = y + (t * parts + part) * width;
    const TZ* gate = z + t * ld_z + part * width;
    auto gated = [&](int j, float* u) {
        float g[V];
        load_pack<float, V>(row + j, u);
        if constexpr (sizeof(TZ) == 4 || V == 1) {
            load_pack<TZ, V>(gate + j, g);
        } else {
            const uint2 r = *reinterpret_cast<const uint2*>(gate + j);
            const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
            g[0] = a.x; g[1] = a.y; g[2] = b.x; g[3] = b.y;
        }
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] *= silu_for<TO>(g[e]);
    };
    float u[HELD][V], sq = 0.f;
#pragma unroll
    for (int n = 0; n < HELD; ++n) {
        const int j = (n * THREADS + me) * V;
        if (j < width) {
            gated(j, u[n]);
#pragma unroll
            for (int e = 0; e < V; ++e) sq = fmaf(u[n][e], u[n][e], sq);
        }
    }
    for (int j = (HELD * THREADS + me) * V; j < width; j += THREADS * V) {
        float v[V];
        gated(j, v);
#pragma unroll
        for (int e = 0; e < V; ++e) sq = fmaf(v[e], v[e], sq);
    }
    sq = THREADS == 32 ? warp_sum(sq) : block_sum(sq, scratch);
    const float inv = 1.f / sqrtf(sq / static_cast<float>(width) + eps);
    const float* w = weight + static_cast<size_t>(part) * width;
    TO* dst = out + (t * parts + part) * width;
    auto finish = [&](int j, const float* v) {
        float f[V], r[V];
        load_pack<float, V>(w + j, f);
#pragma unroll
        for (int e = 0; e < V; ++e) r[e] = __fmul_rn(__fmul_rn(v[e], inv), f[e]);
        if constexpr (sizeof(TO) == 4 || V == 1) {
            store_pack<TO, V>(dst + j, r);
        } else {
            uint2 o;
            o.x = pack_bf16(r[0], r[1]);
            o.y = pack_bf16(r[2], r[3]);
            *reinterpret_cast<uint2*>(dst + j) = o;
        }
    };
#pragma unroll
    for (int n = 0; n < HELD; ++n) {
        const int j = (n * THREADS + me) * V;
        if (j < width) finish(j, u[n]);
    }
    for (int j = (HELD * THREADS + me) * V; j < width; j += THREADS * V) {
        float v[V];
        gated(j, v);
        finish(j, v);
    }
}

template <typename TZ, typename TO>
int launch_group_norm(const float* y, const TZ* z, int ld_z, const float* weight, TO* out, int tokens, int width, int parts, float eps,
                      cudaStream_t stream) {
    const int part = width / parts;
    const long long pairs = static_cast<long long>(tokens) * parts;
    auto aligned = [](const void* q) { return reinterpret_cast<uintptr_t>(q) % 16 == 0; };
    const bool vec = part % 4 == 0 && ld_z % 4 == 0 && aligned(y) && aligned(z) && aligned(weight) && aligned(out);
    const bool wide = part > 1024;
    const long long blocks = wide ? pairs : (pairs + 7) / 8;
    if (blocks > 0x7fffffff) return STRIDE_UNSUPPORTED;
    auto kernel = wide ? (vec ? gated_group_norm_kernel<TZ, TO, 256, 4> : gated_group_norm_kernel<TZ, TO, 256, 1>)
                       : (vec ? gated_group_norm_kernel<TZ, TO, 32, 4> : gated_group_norm_kernel<TZ, TO, 32, 1>);
    stride::launch(kernel, dim3(static_cast<unsigned>(blocks)), dim3(256), 0, stream, y, z, ld_z, weight, out, part, parts, pairs, eps);
    return STRIDE_LAUNCH_STATUS();
}

template <typename TI, typename TO, int V>
int launch_conv(const SsmConvArgs& p, cudaStream_t stream) {
    const int per_row = (p.channels + V - 1) / V, threads = per_row >= 128 ? 128 : (per_row + 31) / 32 * 32;
    const int blocks_x = (per_row + threads - 1) / threads;
    // rows a thread walks: as many as leave every SM a few CTAs
    int run = 16;
    while (run > 1 && static_cast<long long>(blocks_x) * ((p.tokens + run - 1) / run) < 148 * 8) run >>= 1;
    const dim3 grid(blocks_x, (p.tokens + run - 1) / run);
    if (grid.y > 65535) return STRIDE_UNSUPPORTED;
    auto kernel = p.taps == 1   ? ssm_conv_kernel<TI, TO, V, 1>
                  : p.taps == 2 ? ssm_conv_kernel<TI, TO, V, 2>
                  : p.taps == 3 ? ssm_conv_kernel<TI, TO, V, 3>
                  : p.taps == 4 ? ssm_conv_kernel<TI, TO, V, 4>
                                : ssm_conv_kernel<TI, TO, V, 0>;
    stride::launch(kernel, grid, dim3(threads), 0, stream, p, run);
    return STRIDE_LAUNCH_STATUS();
}

inline bool ssm_sizes_ok(int H, int G, int N, int P, int taps) {
    return H > 0 && G > 0 && H % G == 0 && N > 0 && P > 0 && taps > 0;
}

}  // namespace stride

using namespace stride;

extern "C" {

// The first `tokens` rows of u, all of them rows of portions or padding. ring: the state tensor from the ring's first float on.
int stride_ssm_conv(const void* u, int ld, int u_bf16, int channels, int taps, const float* w, const float* b, const float* ring,
                    long long state_stride, const int32_t* seq_of_token, const int32_t* q_start, const int32_t* positions,
                    const int32_t* state_slot, void* out, int ld_out, int tokens, int dtype, cudaStream_t stream) {
    if (tokens < 0 || channels <= 0 || taps <= 0 || ld < channels || ld_out < channels || !w || !b) return STRIDE_BAD_ARGUMENT;
    if (taps > 1 && (!ring || state_stride < static_cast<long long>(taps) * channels)) return STRIDE_BAD_ARGUMENT;
    if (taps > kSsmMaxTaps) return STRIDE_UNSUPPORTED;
    if (tokens == 0) return 0;
    const SsmConvArgs p = {u, ld, channels, taps, w, b, ring, state_stride, seq_of_token, q_start, positions, state_slot, out, ld_out, tokens};
    auto aligned = [](const void* q) { return reinterpret_cast<uintptr_t>(q) % 16 == 0; };
    const bool out_bf16 = dtype == STRIDE_DTYPE_BF16;
    const int pack = out_bf16 ? 8 : 4;
    const bool vec = channels % pack == 0 && ld % 8 == 0 && ld_out % 8 == 0 && aligned(u) && aligned(out) && aligned(w) && aligned(b) &&
                     (taps == 1 || (aligned(ring) && state_stride % 4 == 0));
    if (dtype == STRIDE_DTYPE_F32 && !u_bf16) return vec ? launch_conv<float, float, 4>(p, stream) : launch_conv<float, float, 1>(p, stream);
    if (out_bf16 && u_bf16)
        return vec ? launch_conv<__nv_bfloat16, __nv_bfloat16, 8>(p, stream) : launch_conv<__nv_bfloat16, __nv_bfloat16, 1>(p, stream);
    if (out_bf16) return vec ? launch_conv<float, __nv_bfloat16, 8>(p, stream) : launch_conv<float, __nv_bfloat16, 1>(p, stream);
    return STRIDE_BAD_ARGUMENT;
}

int stride_ssm_tail(const void* u, int ld, int u_bf16, int channels, int taps, float* ring, long long state_stride, const int32_t* q_start,
                    const int32_t* q_len, const int32_t* positions, const int32_t* state_slot, int num_seqs, cudaStream_t stream) {
    if (num_seqs < 0 || channels <= 0 || taps <= 0 || ld < channels || !ring || state_stride < static_cast<long long>(taps) * channels)
        return STRIDE_BAD_ARGUMENT;
    if (taps > kSsmMaxTaps || num_seqs > 65535) return STRIDE_UNSUPPORTED;
    if (num_seqs == 0 || taps == 1) return 0;
    const SsmTailArgs p = {u, ld, u_bf16, channels, taps, ring, state_stride, q_start, q_len, positions, state_slot};
    stride::launch(ssm_tail_kernel, dim3((channels + 127) / 128, num_seqs), dim3(128), 0, stream, p);
    return STRIDE_LAUNCH_STATUS();
}

// One token after the other. x, B, C [tokens, ld] in the compute type behind convolution and SiLU; raw [tokens, ld_raw] float32.
int stride_ssm_scan(const void* x, const void* B, const void* C, int ld, const float* raw, int ld_raw, const float* dt_bias, const float* a_log,
                    const float* skip, float* y, float* state, long long state_stride, const int32_t* q_start, const int32_t* q_len,
                    const int32_t* state_slot, int num_seqs, int H, int G, int N, int P, int dtype, cudaStream_t stream) {
    if (num_seqs < 0 || !ssm_sizes_ok(H, G, N, P, 1) || ld_raw < H || state_stride < static_cast<long long>(H) * N * P) return STRIDE_BAD_ARGUMENT;
    if (dtype != STRIDE_DTYPE_F32 && dtype != STRIDE_DTYPE_BF16) return STRIDE_BAD_ARGUMENT;
    if (num_seqs > 65535 || H > 65535 || N > kSsmMaxState) return STRIDE_UNSUPPORTED;
    if (num_seqs == 0) return 0;
    ScanArgs p = {};
    p.a = C;
    p.k = B;
    p.v = x;
    p.lda = p.ldv = ld;
    p.beta = raw;
    p.ld_beta = ld_raw;
    p.dt_bias = dt_bias;
    p.a_log = a_log;
    p.skip = skip;
    p.o = y;
    p.state = state;
    p.state_stride = state_stride;
    p.q_start = q_start;
    p.q_len = q_len;
    p.state_slot = state_slot;
    p.H = H;
    p.group = H / G;
    p.D = N;
    p.DV = P;
    p.in_bf16 = dtype == STRIDE_DTYPE_BF16 ? 1 : 0;
    return launch_scan<kTokenDecay>(p, num_seqs, stream);
}

// Requests that bring exactly one token each (q_len 0: none). u: the projection before the convolution (float32 or bfloat16).
// Returns -2 for what it does not take (P no multiple of 4, rows off 16-byte boundaries).
int stride_ssm_step(const void* u, int ld, int u_bf16, const float* raw, int ld_raw, const float* w, const float* b, const float* dt_bias,
                    const float* a_log, const float* skip, float* y, float* state, long long state_stride, long long ring_off,
                    const int32_t* q_start, const int32_t* q_len, const int32_t* positions, const int32_t* state_slot, int num_seqs, int H,
                    int G, int N, int P, int taps, cudaStream_t stream) {
    const long long channels = static_cast<long long>(H) * P + 2LL * G * N;
    if (num_seqs < 0 || !ssm_sizes_ok(H, G, N, P, taps) || ld < channels || ld_raw < H || ring_off < static_cast<long long>(H) * N * P ||
        state_stride < ring_off + (taps > 1 ? taps * channels : 0))
        return STRIDE_BAD_ARGUMENT;
    if (num_seqs > 65535 || H > 65535 || N > kSsmMaxState || taps > kSsmMaxTaps || P % 4 || state_stride % 4 || reinterpret_cast<uintptr_t>(state) % 16)
        return STRIDE_UNSUPPORTED;
    if (num_seqs == 0) return 0;
    const SsmStepArgs p = {u, ld, u_bf16, raw, ld_raw, w, b, dt_bias, a_log, skip, y, state, state_stride, ring_off, q_start, q_len, positions,
                           state_slot, H, G, N, P, taps};
    const int cols = P <= 32 ? 32 : P <= 64 ? 64 : 128;
    const dim3 grid((P + cols - 1) / cols, H, num_seqs);
    stride::launch(cols == 32 ? ssm_step_kernel<32> : cols == 64 ? ssm_step_kernel<64> : ssm_step_kernel<128>, grid, dim3(kSsmThreads), 0, stream, p);
    return STRIDE_LAUNCH_STATUS();
}

// Chunk by chunk, bfloat16; moves the tails of the same requests on as well (u: the projection, taps 1: no tails). scratch: float32,
// num_seqs * max_pieces * H * (N * P + 1), max_pieces = ceil(longest portion / 128).
int stride_ssm_chunks(const void* x, const void* B, const void* C, int ld, const float* raw, int ld_raw, const float* dt_bias,
                      const float* a_log, const float* skip, float* y, float* state, long long state_stride, long long ring_off, const void* u,
                      int ld_u, int u_bf16, int taps, const int32_t* q_start, const int32_t* q_len, const int32_t* positions,
                      const int32_t* state_slot, int num_seqs, int H, int G, int N, int P, int max_pieces, float* scratch, cudaStream_t stream) {
    const long long channels = static_cast<long long>(H) * P + 2LL * G * N;
    if (num_seqs < 0 || max_pieces <= 0 || !scratch || !ssm_sizes_ok(H, G, N, P, taps) || ld < channels || ld_u < channels || ld_raw < H ||
        ring_off < static_cast<long long>(H) * N * P || state_stride < ring_off + (taps > 1 ? taps * channels : 0))
        return STRIDE_BAD_ARGUMENT;
    if (static_cast<long long>(num_seqs) * max_pieces > 65535 || H > 65535 || N > kSsmMaxState || reinterpret_cast<uintptr_t>(scratch) % 16)
        return STRIDE_UNSUPPORTED;
    if (num_seqs == 0) return 0;
    auto aligned = [](const void* q) { return reinterpret_cast<uintptr_t>(q) % 16 == 0; };
    SsmChunkArgs p = {};
    p.x = static_cast<const __nv_bfloat16*>(x);
    p.B = static_cast<const __nv_bfloat16*>(B);
    p.C = static_cast<const __nv_bfloat16*>(C);
    p.ld = ld;
    p.raw = raw;
    p.ld_raw = ld_raw;
    p.dt_bias = dt_bias;
    p.a_log = a_log;
    p.skip = skip;
    p.y = y;
    p.piece_s = scratch;
    p.piece_p = scratch + static_cast<size_t>(num_seqs) * max_pieces * H * N * P;
    p.q_start = q_start;
    p.q_len = q_len;
    p.H = H;
    p.G = G;
    p.N = N;
    p.P = P;
    p.max_pieces = max_pieces;
    p.vec = N % 8 == 0 && P % 8 == 0 && ld % 8 == 0 && aligned(x) && aligned(B) && aligned(C);
    const SsmTailArgs tail = {u, ld_u, u_bf16, static_cast<int>(channels), taps, state + ring_off, state_stride, q_start, q_len, positions, state_slot};
    if (N <= 32) return launch_ssm_chunks<32>(p, state, state_stride, state_slot, num_seqs, tail, stream);
    if (N <= 64) return launch_ssm_chunks<64>(p, state, state_stride, state_slot, num_seqs, tail, stream);
    if (N <= 128) return launch_ssm_chunks<128>(p, state, state_stride, state_slot, num_seqs, tail, stream);
    return launch_ssm_chunks<256>(p, state, state_stride, state_slot, num_seqs, tail, stream);
}

// out [tokens, width] = weight * u / sqrt(mean(u^2) + eps), u = y * silu(z), the mean over each of `parts` equal parts of a row.
int stride_gated_group_norm(const float* y, const void* z, int ld_z, int z_bf16, const float* weight, void* out, int tokens, int width,
                            int parts, float eps, int dtype, cudaStream_t stream) {
    if (tokens < 0 || width <= 0 || parts <= 0 || width % parts || ld_z < width) return STRIDE_BAD_ARGUMENT;
    if (tokens == 0) return 0;
    if (dtype == STRIDE_DTYPE_F32 && !z_bf16)
        return launch_group_norm(y, static_cast<const float*>(z), ld_z, weight, static_cast<float*>(out), tokens, width, parts, eps, stream);
    if (dtype == STRIDE_DTYPE_BF16 && z_bf16)
        return launch_group_norm(y, static_cast<const __nv_bfloat16*>(z), ld_z, weight, static_cast<__nv_bfloat16*>(out), tokens, width, parts, eps, stream);
    if (dtype == STRIDE_DTYPE_BF16)
        return launch_group_norm(y, static_cast<const float*>(z), ld_z, weight, static_cast<__nv_bfloat16*>(out), tokens, width, parts, eps, stream);
    return STRIDE_BAD_ARGUMENT;
}

}  // extern "C"

// Mixers that keep a matrix per head as their memory: S [D, DV] in float32, updated once a token by a rank-one term and
// read with a query. Two rules:
//
//   gated delta rule     S <- diag(g_t) S ;  u = beta_t (v_t - S^T k_t) ;  S <- S + k_t u^T ;  o_t = S^T q_t
//                        (Yang, Kautz, Hatamizadeh, "Gated Delta Networks: Improving Mamba2 with Delta Rule"; here the
//                        decay g_t is a vector over the D key channels)
//   decayed memory with a bonus (the time mixing of RWKV-6: Peng et al., "Eagle and Finch: RWKV with Matrix-Valued
//                        States and Dynamic Recurrence")
//                        o_t = (S + diag(b) k_t v_t^T)^T r_t ;  S <- diag(w_t) S + k_t v_t^T
//
// Both are independent over the DV columns of S, and along a column the only coupling is one sum over D per read. The
// scan kernel gives a column to 4, 8 or 16 neighbouring lanes: each holds R of the rows in registers (groups of four
// neighbouring rows; rows beyond D carry zeros), sums its part in four partial sums and the lanes add up by shuffles,
// always in the same order. A CTA of 128 threads owns 32, 16 or 8 columns of one head of one request and walks the
// request's tokens of the step in order; the inputs of 8 or 16 tokens are staged in shared memory at a time, the next ones
// being fetched into registers meanwhile. The order of every sum depends on the token
// only, so a token's output is bitwise the same in a whole prompt, in portions or decoded alone. State per request lives
// in one float32 row of the mixer's state tensor: S [heads, D, DV], then whatever the mixer needs of the past inputs.
//
// Kernels around the scans:
//   delta_prepare   per token: causal convolution (taps from the state's tail at a portion's start) and SiLU of the q, k
//                   and v projections, unit length for q and k per head (q also times D^-1/2), beta = sigmoid, and the
//                   decay exp(-exp(A_log) softplus(a + dt_bias)); everything float32
//   shift_mix       per token: the lerps between a token's input and the previous token's (the state's at a portion's
//                   start), one per consumer; the portion's last input goes into the state
//   head_norm_gate  o / rms(o) * weight * gate per head, into the compute type for the output projection
// The scans end by writing S back and, for the delta rule, by moving the convolution's tail in the state forward.
#include "memory_scan.cuh"

namespace stride {

// ------------------------------------------------------------------------------------------------ delta_prepare
// proj [tokens, ld] (compute type): columns [0, GD) q, [GD, 2GD) k, [2GD, 2GD + HV) v, then H columns of beta's
// projection. conv_w [C, taps] float32 for the C = 2GD + HV channels in the same order. low [tokens, ld_low] float32:
// columns [0, HD) the decay's projection. tail: the state's rows [taps - 1, C] at `tail_off` floats into a slot's row.
// Outputs float32: qk [tokens, 2GD] (q then k, unit length), v [tokens, HV], beta [tokens, H], decay [tokens, HD].
// What is handed on of a decay g is g - 1 = expm1(log g), and the scans compute S + (g - 1) S: for a channel that forgets
// slowly g is within 1e-4 of 1, where float32 has steps of 6e-8 and a rounded g costs a little with every token.
// One warp a head: warps 0..2G-1 the q and k heads, then H warps for the v heads, which also do beta and the decay.
constexpr int kPrepWarps = 8;
constexpr int kMaxPerLane = 8;      // head sizes up to 256

template <typename T>
__global__ void __launch_bounds__(kPrepWarps * 32)
delta_prepare_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ conv_w, const float* __restrict__ low, int ld_low,
                     const float* __restrict__ a_log, const float* __restrict__ dt_bias, const float* __restrict__ state,
                     long long state_stride, long long tail_off, const int32_t* __restrict__ seq_of_token,
                     const int32_t* __restrict__ q_start, const int32_t* __restrict__ state_slot, float* __restrict__ qk,
                     float* __restrict__ v_out, float* __restrict__ beta, float* __restrict__ decay, int G, int H, int D, int DV,
                     int taps, float unit_eps) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y * kPrepWarps + warp;
    if (head >= 2 * G + H) return;
    const int GD = G * D, HV = H * DV, C = 2 * GD + HV;
    const bool is_v = head >= 2 * G;
    const int n = is_v ? DV : D;
    const int c0 = is_v ? 2 * GD + (head - 2 * G) * DV : head * D;       // first channel of this head
    const int seq = seq_of_token[t];
    float* dst = is_v ? v_out + static_cast<size_t>(t) * HV + (head - 2 * G) * DV : qk + static_cast<size_t>(t) * 2 * GD + head * D;
    if (seq < 0) {          // a padded row of a fixed-size batch
        for (int e = lane; e < n; e += 32) dst[e] = 0.f;
        if (is_v) {
            const int h = head - 2 * G;
            for (int e = lane; e < D; e += 32) decay[static_cast<size_t>(t) * H * D + h * D + e] = 0.f;
            if (lane == 0) beta[static_cast<size_t>(t) * H + h] = 0.f;
        }
        return;
    }
    const int start = q_start[seq];
    const int local = t - start;
    const float* tail = state + static_cast<size_t>(state_slot[seq]) * state_stride + tail_off;
    float y[kMaxPerLane];
    float ss = 0.f;
#pragma unroll
    for (int r = 0; r < kMaxPerLane; ++r) {
        const int e = lane + 32 * r;
        y[r] = 0.f;
        if (e < n) {
            const int c = c0 + e;
            float acc = 0.f;
            for (int j = 0; j < taps; ++j) {
                const int src = local - (taps - 1) + j;
                const float x = src >= 0 ? to_f32(proj[static_cast<size_t>(start + src) * ld + c])
                                         : tail[static_cast<size_t>(taps - 1 + src) * C + c];
                acc = fmaf(conv_w[static_cast<size_t>(c) * taps + j], x, acc);
            }
            y[r] = silu_f(acc);
            ss = fmaf(y[r], y[r], ss);
        }
    }
    float mult = 1.f;
    if (!is_v) {
        ss = warp_sum(ss);
        mult = 1.f / sqrtf(ss + unit_eps);
        if (head < G) mult *= 1.f / sqrtf(static_cast<float>(D));
    }
#pragma unroll
    for (int r = 0; r < kMaxPerLane; ++r) {
        const int e = lane + 32 * r;
        if (e < n) dst[e] = y[r] * mult;
    }
    if (is_v) {
        const int h = head - 2 * G;
        const float rate = expf(a_log[h]);
        for (int e = lane; e < D; e += 32) {
            const float a = low[static_cast<size_t>(t) * ld_low + h * D + e] + dt_bias[h * D + e];
            decay[static_cast<size_t>(t) * H * D + h * D + e] = expm1f(-rate * softplus_f(a));
        }
        if (lane == 0) beta[static_cast<size_t>(t) * H + h] = sigmoid_f(to_f32(proj[static_cast<size_t>(t) * ld + C + h]));
    }
}

// ---------------------------------------------------------------------------------------------------- shift_mix
// x [tokens, width] (compute type); mu [mixes, width] float32; out [mixes, tokens, width] (compute type):
// out[s, t] = x[t] + (prev - x[t]) * mu[s], prev = x[t - 1] inside a portion and the state's vector at its start. The CTA
// of a portion's first token then stores the portion's last input as the new state (it alone touches the state).
template <typename T>
__global__ void __launch_bounds__(256)
shift_mix_kernel(const T* __restrict__ x, const float* __restrict__ mu, float* __restrict__ state, long long state_stride,
                 long long prev_off, const int32_t* __restrict__ seq_of_token, const int32_t* __restrict__ q_start,
                 const int32_t* __restrict__ q_len, const int32_t* __restrict__ state_slot, T* __restrict__ out, int tokens, int width,
                 int mixes) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const int seq = seq_of_token[t];
    if (seq < 0) {
        for (int c = threadIdx.x; c < width; c += blockDim.x)
            for (int s = 0; s < mixes; ++s) out[(static_cast<size_t>(s) * tokens + t) * width + c] = from_f32<T>(0.f);
        return;
    }
    const int start = q_start[seq];
    const bool first = t == start;
    float* prev_state = state + static_cast<size_t>(state_slot[seq]) * state_stride + prev_off;
    const T* last = x + static_cast<size_t>(start + q_len[seq] - 1) * width;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const float cur = to_f32(x[static_cast<size_t>(t) * width + c]);
        const float prev = first ? prev_state[c] : to_f32(x[static_cast<size_t>(t - 1) * width + c]);
        const float d = prev - cur;
        for (int s = 0; s < mixes; ++s)
            out[(static_cast<size_t>(s) * tokens + t) * width + c] = from_f32<T>(fmaf(d, mu[static_cast<size_t>(s) * width + c], cur));
        if (first) prev_state[c] = to_f32(last[c]);
    }
}

// ------------------------------------------------------------------------------------------------ head_norm_gate
// o [tokens, H, DV] float32 -> out [tokens, H * DV] (compute type): o / sqrt(mean(o^2) + eps) * weight * gate.
// weight [.. ] float32 read at h * w_head_stride + j (0: one weight for all heads). gate_kind 0: sigmoid of float32
// gate[t * ld_gate + h * DV + j]; 1: silu of a compute-type gate at the same place; 2: sigmoid of a compute-type gate.
// One warp a (token, head); V columns a lane and turn (4 where rows and pointers allow 16-byte accesses).
template <typename T, int V>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ weight, int w_head_stride, const void* __restrict__ gate,
                      int ld_gate, int gate_kind, T* __restrict__ out, int tokens, int H, int DV, float eps) {
    pdl_trigger();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long pair = static_cast<long long>(blockIdx.x) * 8 + warp;
    if (pair >= static_cast<long long>(tokens) * H) return;
    const int t = static_cast<int>(pair / H), h = static_cast<int>(pair % H);
    const float* row = o + (static_cast<size_t>(t) * H + h) * DV;
    const size_t g0 = static_cast<size_t>(t) * ld_gate + h * DV;
    struct alignas(V * sizeof(T)) Pack { T v[V]; };
    float ss = 0.f;
    for (int j = lane * V; j < DV; j += 32 * V) {
        alignas(16) float x[V];
        if constexpr (V == 4) *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(row + j);
        else x[0] = row[j];
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(x[e], x[e], ss);
    }
    ss = warp_sum(ss);
    const float inv = 1.f / sqrtf(ss / static_cast<float>(DV) + eps);
    for (int j = lane * V; j < DV; j += 32 * V) {
        alignas(16) float x[V];
        alignas(16) float w[V];
        Pack g, y;
        if constexpr (V == 4) {
            *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(row + j);
            *reinterpret_cast<float4*>(w) = *reinterpret_cast<const float4*>(weight + h * w_head_stride + j);
        } else {
            x[0] = row[j];
            w[0] = weight[h * w_head_stride + j];
        }
        if (gate_kind) g = *reinterpret_cast<const Pack*>(static_cast<const T*>(gate) + g0 + j);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            const float z = gate_kind ? to_f32(g.v[e]) : static_cast<const float*>(gate)[g0 + j + e];
            y.v[e] = from_f32<T>(x[e] * inv * w[e] * (gate_kind == 1 ? silu_f(z) : sigmoid_f(z)));
        }
        *reinterpret_cast<Pack*>(out + (static_cast<size_t>(t) * H + h) * DV + j) = y;
    }
}

// The same with a CTA a (token, head), for heads so wide that a warp would walk them for long (one norm over all heads of a
// token counts as one head). V columns a thread and turn.
template <typename T, int V>
__global__ void __launch_bounds__(256)
head_norm_gate_wide_kernel(const float* __restrict__ o, const float* __restrict__ weight, int w_head_stride, const void* __restrict__ gate,
                           int ld_gate, int gate_kind, T* __restrict__ out, int H, int DV, float eps) {
    __shared__ float scratch[32];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x / H, h = blockIdx.x % H;
    const float* row = o + (static_cast<size_t>(t) * H + h) * DV;
    const size_t g0 = static_cast<size_t>(t) * ld_gate + h * DV;
    float ss = 0.f;
    for (int j = threadIdx.x * V; j < DV; j += blockDim.x * V) {
        alignas(16) float x[V];
        if constexpr (V == 4) *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(row + j);
        else x[0] = row[j];
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(x[e], x[e], ss);
    }
    const float inv = 1.f / sqrtf(block_sum(ss, scratch) / static_cast<float>(DV) + eps);
    for (int j = threadIdx.x * V; j < DV; j += blockDim.x * V) {
        alignas(16) float x[V];
        alignas(16) float w[V];
        alignas(16) T g[V];
        alignas(16) T y[V];
        if constexpr (V == 4) {
            *reinterpret_cast<float4*>(x) = *reinterpret_cast<const float4*>(row + j);
            *reinterpret_cast<float4*>(w) = *reinterpret_cast<const float4*>(weight + h * w_head_stride + j);
        } else {
            x[0] = row[j];
            w[0] = weight[h * w_head_stride + j];
        }
        struct alignas(V * sizeof(T)) Pack { T v[V]; };
        if (gate_kind) *reinterpret_cast<Pack*>(g) = *reinterpret_cast<const Pack*>(static_cast<const T*>(gate) + g0 + j);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            const float z = gate_kind ? to_f32(g[e]) : static_cast<const float*>(gate)[g0 + j + e];
            y[e] = from_f32<T>(x[e] * inv * w[e] * (gate_kind == 1 ? silu_f(z) : sigmoid_f(z)));
        }
        *reinterpret_cast<Pack*>(out + (static_cast<size_t>(t) * H + h) * DV + j) = *reinterpret_cast<Pack*>(y);
    }
}

constexpr int kWideHead = 512;

// Between the two passes over pieces of the delta rule, whose pieces carry a memory across by a full matrix: piece_t [z, H, D, D] holds it, piece_s
// [z, H, D, DV] what the piece adds from a zero memory; S_next = T S + B. A CTA owns 16 columns of S of one head of one
// request and walks the pieces in order; T comes through shared memory in slabs of 16 columns. The memory at a piece's
// start takes the place of the piece's own sum, the memory after the last piece goes into the state.
constexpr int kCombineCols = 16, kCombineThreads = 256, kCombineMaxD = 256;

__global__ void __launch_bounds__(kCombineThreads)
delta_pieces_combine_kernel(float* __restrict__ piece_s, const float* __restrict__ piece_t, float* __restrict__ state,
                            long long state_stride, const int32_t* __restrict__ q_len, const int32_t* __restrict__ state_slot, int H, int D,
                            int DV, int piece, int max_pieces) {
    pdl_trigger();
    pdl_wait();
    constexpr int PER = kCombineMaxD * kCombineCols / kCombineThreads;       // entries of the CTA's columns a thread, at most
    __shared__ float S_s[kCombineMaxD][kCombineCols], T_s[kCombineMaxD][kCombineCols + 1];
    const int seq = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kCombineCols;
    const int len = q_len[seq];
    if (len <= 0) return;
    float* S_g = state + static_cast<size_t>(state_slot[seq]) * state_stride + static_cast<size_t>(h) * D * DV;
    const int entries = D * kCombineCols;
    for (int idx = threadIdx.x; idx < entries; idx += kCombineThreads) {
        const int row = idx / kCombineCols, col = idx % kCombineCols;
        S_s[row][col] = c0 + col < DV ? S_g[static_cast<size_t>(row) * DV + c0 + col] : 0.f;
    }
    __syncthreads();
    const int pieces = (len + piece - 1) / piece;
    for (int c = 0; c < pieces; ++c) {
        const size_t z = static_cast<size_t>(seq) * max_pieces + c;
        const float* T = piece_t + (z * H + h) * D * D;
        float* B = piece_s + (z * H + h) * D * DV;
        float acc[PER];
#pragma unroll
        for (int n = 0; n < PER; ++n) acc[n] = 0.f;
        for (int k0 = 0; k0 < D; k0 += kCombineCols) {
            for (int idx = threadIdx.x; idx < entries; idx += kCombineThreads) {
                const int row = idx / kCombineCols, kk = idx % kCombineCols;
                T_s[row][kk] = k0 + kk < D ? T[static_cast<size_t>(row) * D + k0 + kk] : 0.f;
            }
            __syncthreads();
#pragma unroll
            for (int n = 0; n < PER; ++n) {
                const int idx = n * kCombineThreads + threadIdx.x;
                if (idx < entries) {
                    const int row = idx / kCombineCols, col = idx % kCombineCols;
#pragma unroll
                    for (int kk = 0; kk < kCombineCols; ++kk)
                        if (k0 + kk < D) acc[n] = fmaf(T_s[row][kk], S_s[k0 + kk][col], acc[n]);
                }
            }
            __syncthreads();
        }
#pragma unroll
        for (int n = 0; n < PER; ++n) {
            const int idx = n * kCombineThreads + threadIdx.x;
            if (idx < entries) {
                const int row = idx / kCombineCols, col = idx % kCombineCols;
                if (c0 + col < DV) {
                    float* at = B + static_cast<size_t>(row) * DV + c0 + col;
                    const float own = *at;
                    *at = S_s[row][col];                // every thread reads and writes its own entries only
                    acc[n] += own;
                }
            }
        }
        __syncthreads();
#pragma unroll
        for (int n = 0; n < PER; ++n) {
            const int idx = n * kCombineThreads + threadIdx.x;
            if (idx < entries) S_s[idx / kCombineCols][idx % kCombineCols] = acc[n];
        }
        __syncthreads();
    }
    for (int idx = threadIdx.x; idx < entries; idx += kCombineThreads) {
        const int row = idx / kCombineCols, col = idx % kCombineCols;
        if (c0 + col < DV) S_g[static_cast<size_t>(row) * DV + c0 + col] = S_s[row][col];
    }
}

}  // namespace stride

using namespace stride;

extern "C" {

int stride_delta_prepare(const void* proj, int ld, const float* conv_w, const float* low, int ld_low, const float* a_log,
                         const float* dt_bias, const float* state, long long state_stride, long long tail_off,
                         const int32_t* seq_of_token, const int32_t* q_start, const int32_t* state_slot, float* qk, float* v_out,
                         float* beta, float* decay, int tokens, int G, int H, int D, int DV, int taps, float unit_eps, int dtype,
                         cudaStream_t stream) {
    if (tokens < 0 || G <= 0 || H <= 0 || D <= 0 || DV <= 0 || taps <= 0 || H % G) return STRIDE_BAD_ARGUMENT;
    if (D > 32 * kMaxPerLane || DV > 32 * kMaxPerLane) return STRIDE_UNSUPPORTED;
    if (tokens == 0) return 0;
    const dim3 grid(tokens, (2 * G + H + kPrepWarps - 1) / kPrepWarps), block(kPrepWarps * 32);
    if (dtype == STRIDE_DTYPE_F32)
        stride::launch(delta_prepare_kernel<float>, grid, block, 0, stream, static_cast<const float*>(proj), ld, conv_w, low, ld_low, a_log,
                       dt_bias, state, state_stride, tail_off, seq_of_token, q_start, state_slot, qk, v_out, beta, decay, G, H, D, DV, taps,
                       unit_eps);
    else if (dtype == STRIDE_DTYPE_BF16)
        stride::launch(delta_prepare_kernel<__nv_bfloat16>, grid, block, 0, stream, static_cast<const __nv_bfloat16*>(proj), ld, conv_w, low,
                       ld_low, a_log, dt_bias, state, state_stride, tail_off, seq_of_token, q_start, state_slot, qk, v_out, beta, decay, G, H,
                       D, DV, taps, unit_eps);
    else
        return STRIDE_BAD_ARGUMENT;
    return STRIDE_LAUNCH_STATUS();
}

// The gated delta rule over the step's requests. qk, v, beta, decay: what delta_prepare wrote. proj: the projections
// whose last taps - 1 rows become the convolution's new tail.
// piece > 0: in pieces of that many tokens, parallel over the pieces (every piece from a zero memory; every piece's matrix;
// the memories at the pieces' starts; every piece from its start). scratch: float32, at least
// num_seqs * max_pieces * H * D * (DV + D). As for the other rule, the sums then take another order than the chain's.
int stride_delta_scan(const float* qk, const float* v, const float* beta, const float* decay, float* o, float* state,
                      long long state_stride, long long tail_off, const void* proj, int ld_proj, const int32_t* q_start,
                      const int32_t* q_len, const int32_t* state_slot, int num_seqs, int G, int H, int D, int DV, int taps, int dtype,
                      int piece, int max_pieces, float* scratch, cudaStream_t stream) {
    if (num_seqs < 0 || G <= 0 || H <= 0 || D <= 0 || DV <= 0 || taps <= 0 || H % G) return STRIDE_BAD_ARGUMENT;
    if (piece < 0 || (piece > 0 && (max_pieces <= 0 || scratch == nullptr))) return STRIDE_BAD_ARGUMENT;
    if (piece > 0 && D > kCombineMaxD) return STRIDE_UNSUPPORTED;
    if (dtype != STRIDE_DTYPE_F32 && dtype != STRIDE_DTYPE_BF16) return STRIDE_BAD_ARGUMENT;
    if (num_seqs == 0) return 0;
    ScanArgs p = {};
    p.a = qk;
    p.k = qk + static_cast<size_t>(G) * D;
    p.lda = 2 * G * D;
    p.w = decay;
    p.v = v;
    p.ldv = H * DV;
    p.beta = beta;
    p.o = o;
    p.state = state;
    p.state_stride = state_stride;
    p.q_start = q_start;
    p.q_len = q_len;
    p.state_slot = state_slot;
    p.H = H;
    p.group = H / G;
    p.D = D;
    p.DV = DV;
    p.in_bf16 = 0;
    p.proj = proj;
    p.ld_proj = ld_proj;
    p.C = 2 * G * D + H * DV;
    p.taps = taps;
    p.tail_off = tail_off;
    p.proj_bf16 = dtype == STRIDE_DTYPE_BF16 ? 1 : 0;      // the tail is read in the projections' type, the rest is float32
    if (piece == 0) return launch_scan<0>(p, num_seqs, stream);
    const size_t zs = static_cast<size_t>(num_seqs) * max_pieces;
    float* piece_s = scratch;
    float* piece_t = scratch + zs * H * D * DV;
    p.piece = piece;
    p.max_pieces = max_pieces;
    p.mode = 1;
    p.init = 1;
    p.piece_s = piece_s;
    int code = launch_scan<0>(p, num_seqs, stream);             // what every piece adds from a zero memory
    if (code != 0) return code;
    ScanArgs t = p;
    t.v = nullptr;
    t.DV = D;
    t.init = 2;
    t.piece_s = piece_t;
    code = launch_scan<0>(t, num_seqs, stream);                 // every piece's matrix
    if (code != 0) return code;
    stride::launch(delta_pieces_combine_kernel, dim3((DV + kCombineCols - 1) / kCombineCols, H, num_seqs), dim3(kCombineThreads), 0, stream,
                   piece_s, static_cast<const float*>(piece_t), state, state_stride, q_len, state_slot, H, D, DV, piece, max_pieces);
    code = STRIDE_LAUNCH_STATUS();
    if (code != 0) return code;
    p.mode = 2;
    return launch_scan<0>(p, num_seqs, stream);                 // every piece from its start, with the outputs
}

// Decayed memory with a bonus. r, k, v [tokens, H * D] in the compute type (one head size for keys and values);
// wlog [tokens, H * D] float32: the decay is exp(-exp(wlog + w0)).
// piece > 0: the recurrence in pieces of that many tokens, parallel over the pieces (three launches: every piece from a zero
// memory; the memories at the pieces' starts; every piece from its start). scratch: float32, at least
// num_seqs * max_pieces * H * D * (D + 1), max_pieces = ceil(longest portion / piece). The sums then take another order than
// the single chain's, so the result depends on the cutting in the last bits: for bfloat16 runs and long portions.
int stride_bonus_scan(const void* r, const void* k, const void* v, const float* wlog, const float* w0, const float* bonus, float* o,
                      float* state, long long state_stride, const int32_t* q_start, const int32_t* q_len, const int32_t* state_slot,
                      int num_seqs, int H, int D, int dtype, int piece, int max_pieces, float* scratch, cudaStream_t stream) {
    if (num_seqs < 0 || H <= 0 || D <= 0 || piece < 0 || (piece > 0 && (max_pieces <= 0 || scratch == nullptr))) return STRIDE_BAD_ARGUMENT;
    if (dtype != STRIDE_DTYPE_F32 && dtype != STRIDE_DTYPE_BF16) return STRIDE_BAD_ARGUMENT;
    if (num_seqs == 0) return 0;
    ScanArgs p = {};
    p.a = r;
    p.k = k;
    p.lda = H * D;
    p.w = wlog;
    p.w0 = w0;
    p.bonus = bonus;
    p.v = v;
    p.ldv = H * D;
    p.o = o;
    p.state = state;
    p.state_stride = state_stride;
    p.q_start = q_start;
    p.q_len = q_len;
    p.state_slot = state_slot;
    p.H = H;
    p.group = 1;
    p.D = D;
    p.DV = D;
    p.in_bf16 = dtype == STRIDE_DTYPE_BF16 ? 1 : 0;
    p.taps = 0;
    if (piece == 0) return launch_scan<1>(p, num_seqs, stream);
    p.piece = piece;
    p.max_pieces = max_pieces;
    p.piece_s = scratch;
    p.piece_p = scratch + static_cast<size_t>(num_seqs) * max_pieces * H * D * D;
    p.mode = 1;
    int code = launch_scan<1>(p, num_seqs, stream);
    if (code != 0) return code;
    const int entries = H * D * D;
    stride::launch(pieces_combine_kernel, dim3((entries + 255) / 256, num_seqs), dim3(256), 0, stream, p.piece_s,
                   static_cast<const float*>(p.piece_p), state, state_stride, q_len, state_slot, H, D, D, piece, max_pieces);
    code = STRIDE_LAUNCH_STATUS();
    if (code != 0) return code;
    p.mode = 2;
    return launch_scan<1>(p, num_seqs, stream);
}

int stride_shift_mix(const void* x, const float* mu, float* state, long long state_stride, long long prev_off,
                     const int32_t* seq_of_token, const int32_t* q_start, const int32_t* q_len, const int32_t* state_slot, void* out,
                     int tokens, int width, int mixes, int dtype, cudaStream_t stream) {
    if (tokens < 0 || width <= 0 || mixes <= 0) return STRIDE_BAD_ARGUMENT;
    if (tokens == 0) return 0;
    if (dtype == STRIDE_DTYPE_F32)
        stride::launch(shift_mix_kernel<float>, dim3(tokens), dim3(256), 0, stream, static_cast<const float*>(x), mu, state, state_stride,
                       prev_off, seq_of_token, q_start, q_len, state_slot, static_cast<float*>(out), tokens, width, mixes);
    else if (dtype == STRIDE_DTYPE_BF16)
        stride::launch(shift_mix_kernel<__nv_bfloat16>, dim3(tokens), dim3(256), 0, stream, static_cast<const __nv_bfloat16*>(x), mu, state,
                       state_stride, prev_off, seq_of_token, q_start, q_len, state_slot, static_cast<__nv_bfloat16*>(out), tokens, width,
                       mixes);
    else
        return STRIDE_BAD_ARGUMENT;
    return STRIDE_LAUNCH_STATUS();
}

int stride_head_norm_gate(const float* o, const float* weight, int w_head_stride, const void* gate, int ld_gate, int gate_kind, void* out,
                          int tokens, int H, int DV, float eps, int dtype, cudaStream_t stream) {
    if (tokens < 0 || H <= 0 || DV <= 0 || gate_kind < 0 || gate_kind > 2) return STRIDE_BAD_ARGUMENT;
    if (tokens == 0) return 0;
    if (dtype != STRIDE_DTYPE_F32 && dtype != STRIDE_DTYPE_BF16) return STRIDE_BAD_ARGUMENT;
    const long long pairs = static_cast<long long>(tokens) * H;
    if (pairs >= 0x7fffffff) return STRIDE_UNSUPPORTED;
    auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
    const bool vec = DV % 4 == 0 && ld_gate % 4 == 0 && aligned(o) && aligned(weight) && aligned(gate) && aligned(out) && w_head_stride % 4 == 0;
    if (DV >= kWideHead) {
        const dim3 cta(DV / (vec ? 4 : 1) >= 256 ? 256 : 128), each(static_cast<unsigned>(pairs));
        if (dtype == STRIDE_DTYPE_F32)
            stride::launch(vec ? head_norm_gate_wide_kernel<float, 4> : head_norm_gate_wide_kernel<float, 1>, each, cta, 0, stream, o, weight,
                           w_head_stride, gate, ld_gate, gate_kind, static_cast<float*>(out), H, DV, eps);
        else
            stride::launch(vec ? head_norm_gate_wide_kernel<__nv_bfloat16, 4> : head_norm_gate_wide_kernel<__nv_bfloat16, 1>, each, cta, 0,
                           stream, o, weight, w_head_stride, gate, ld_gate, gate_kind, static_cast<__nv_bfloat16*>(out), H, DV, eps);
        return STRIDE_LAUNCH_STATUS();
    }
    const dim3 grid(static_cast<unsigned>((pairs + 7) / 8)), block(256);
    if (dtype == STRIDE_DTYPE_F32)
        stride::launch(vec ? head_norm_gate_kernel<float, 4> : head_norm_gate_kernel<float, 1>, grid, block, 0, stream, o, weight, w_head_stride,
                       gate, ld_gate, gate_kind, static_cast<float*>(out), tokens, H, DV, eps);
    else
        stride::launch(vec ? head_norm_gate_kernel<__nv_bfloat16, 4> : head_norm_gate_kernel<__nv_bfloat16, 1>, grid, block, 0, stream, o, weight,
                       w_head_stride, gate, ld_gate, gate_kind, static_cast<__nv_bfloat16*>(out), tokens, H, DV, eps);
    return STRIDE_LAUNCH_STATUS();
}

}  // extern "C"

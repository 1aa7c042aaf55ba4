// The experts' products of a routed feed-forward for steps of a few tokens (decoding), bfloat16, where the time goes into
// reading the chosen experts' weights once:
//   C[p, :] = act(A[src(p), :] W[e(p)]^T)   for the rows p of every expert e.
// Either rows lie expert by expert (`offsets`, a plan's), or there is no plan: row p is (token, choice) pair p, which belongs to
// expert ids[p], and every CTA picks its expert's pairs out of the list itself (`pairs` of them, up to 512; src(p) = p / top).
//
// A CTA takes 16 rows of one expert's weights and all of K, its four warps every fourth block of 32 columns. The weights are the
// 16-row operand of mma.sync m16n8k16 and go from global memory straight into fragments, 16 bytes a lane and row: a lane's eight
// neighbouring columns are the k-places of two products, and the tokens' rows are read with the same assignment, so the sums
// are those of the columns in another order. Eight 16-byte loads of weights a lane are in flight at a time. The tokens of an
// expert are the 8-column operand, up to 32 of them at a time (more: the CTA walks the expert's rows in turns and reads its
// weights again, from L2). The warps' sums meet in shared memory, where the activation is applied. A CTA whose expert has no rows
// leaves at once.
//
// act 0 to 3 and row_weight as in moe.cu. The order of a row's sums depends on K only.
#include "common.cuh"
#include "mma.cuh"

namespace stride {

constexpr int kStreamWarps = 4;
constexpr int kStreamRows = 16;          // weight rows a CTA
constexpr int kStreamTokens = 32;        // rows of A a turn
constexpr int kStreamMaxPairs = 512;
constexpr int kStreamAhead = 4;          // blocks of 32 columns whose weights a warp asks for together

__device__ __forceinline__ float stream_pair(int act, float g, float u, float limit, float alpha) {
    if (act == 3) return g / (1.f + expf(-g)) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}

// NT tiles of 8 tokens; src: this lane's token of each tile (null: none).
template <int NT>
__device__ __forceinline__ void stream_rows(const __nv_bfloat16* w_lo, const __nv_bfloat16* w_hi, const __nv_bfloat16* const* src, int K, int warp,
                                            int tg, float (&acc)[4][4]) {
    const int blocks = (K + 31) / 32;
    for (int b0 = warp; b0 < blocks; b0 += kStreamWarps * kStreamAhead) {
        uint4 lo[kStreamAhead], hi[kStreamAhead];
#pragma unroll
        for (int i = 0; i < kStreamAhead; ++i) {
            const int k = (b0 + i * kStreamWarps) * 32 + tg * 8;
            lo[i] = hi[i] = make_uint4(0, 0, 0, 0);
            if (k < K) {        // K is a multiple of 8
                if (w_lo) lo[i] = __ldg(reinterpret_cast<const uint4*>(w_lo + k));
                if (w_hi) hi[i] = __ldg(reinterpret_cast<const uint4*>(w_hi + k));
            }
        }
#pragma unroll
        for (int i = 0; i < kStreamAhead; ++i) {
            const int k = (b0 + i * kStreamWarps) * 32 + tg * 8;
            const uint32_t a0[4] = {lo[i].x, hi[i].x, lo[i].y, hi[i].y}, a1[4] = {lo[i].z, hi[i].z, lo[i].w, hi[i].w};
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                uint4 b = make_uint4(0, 0, 0, 0);
                if (src[n] && k < K) b = *reinterpret_cast<const uint4*>(src[n] + k);
                mma_bf16_16816(acc[n], a0, b.x, b.y);
                mma_bf16_16816(acc[n], a1, b.z, b.w);
            }
        }
    }
}

template <typename OutT>
__global__ void __launch_bounds__(kStreamWarps * 32)
moe_stream_kernel(const __nv_bfloat16* __restrict__ A, int lda, const int32_t* __restrict__ row_map, const __nv_bfloat16* __restrict__ W,
                  const int32_t* __restrict__ offsets, const int32_t* __restrict__ ids, int pairs, int top, OutT* __restrict__ C, int ldc, int N, int K,
                  int act, float limit, float alpha, const float* __restrict__ row_weight) {
    __shared__ float red[kStreamWarps][kStreamRows][kStreamTokens + 1];
    __shared__ int picked[kStreamMaxPairs];
    pdl_trigger();
    pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tg = lane & 3;
    const int e = blockIdx.y;
    int lo = 0, hi = 0;
    if (ids) {              // this expert's pairs in ascending order; every warp finds (and notes) all of them, so nobody waits
        for (int p0 = 0; p0 < pairs; p0 += 128) {
            int own[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) own[i] = p0 + i * 32 + lane < pairs ? ids[p0 + i * 32 + lane] : -1;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                if (p0 + i * 32 >= pairs) break;
                const unsigned mine = __ballot_sync(0xffffffffu, own[i] == e);
                if ((mine >> lane) & 1u) picked[hi + __popc(mine & ((1u << lane) - 1u))] = p0 + i * 32 + lane;
                hi += __popc(mine);
            }
        }
        if (hi == 0) return;
        __syncwarp();
    } else {
        lo = offsets[e];
        hi = offsets[e + 1];
        if (lo >= hi) return;
    }
    auto row_at = [&](int p) { return ids ? picked[p] : p; };
    const int n0 = blockIdx.x * kStreamRows;
    const __nv_bfloat16* We = W + (static_cast<size_t>(e) * N + n0) * K;
    const __nv_bfloat16* w_lo = n0 + g < N ? We + static_cast<size_t>(g) * K : nullptr;
    const __nv_bfloat16* w_hi = n0 + g + 8 < N ? We + static_cast<size_t>(g + 8) * K : nullptr;
    for (int p0 = lo; p0 < hi; p0 += kStreamTokens) {
        const int rows = min(hi - p0, kStreamTokens);
        const __nv_bfloat16* src[4];
#pragma unroll
        for (int n = 0; n < 4; ++n) {
            const int p = p0 + n * 8 + g;
            src[n] = nullptr;
            if (n * 8 + g < rows) src[n] = A + static_cast<size_t>(ids ? picked[p] / top : row_map ? row_map[p] : p) * lda;
        }
        float acc[4][4];
#pragma unroll
        for (int n = 0; n < 4; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
        if (rows <= 8) stream_rows<1>(w_lo, w_hi, src, K, warp, tg, acc);
        else if (rows <= 16) stream_rows<2>(w_lo, w_hi, src, K, warp, tg, acc);
        else stream_rows<4>(w_lo, w_hi, src, K, warp, tg, acc);
        if (p0 > lo) __syncthreads();           // the turn before has been read
#pragma unroll
        for (int n = 0; n < 4; ++n)
            if (n * 8 < rows) {
#pragma unroll
                for (int x = 0; x < 4; ++x) red[warp][g + 8 * (x >> 1)][n * 8 + 2 * tg + (x & 1)] = acc[n][x];
            }
        __syncthreads();
        auto sum = [&](int r, int t) {
            float v = 0.f;
#pragma unroll
            for (int w = 0; w < kStreamWarps; ++w) v += red[w][r][t];
            return row_weight ? v * row_weight[row_at(p0 + t)] : v;
        };
        if (act >= 2) {                         // rows 2i and 2i + 1: gate and up of a unit
            for (int i = threadIdx.x; i < kStreamRows / 2 * rows; i += blockDim.x) {
                const int unit = i % (kStreamRows / 2), t = i / (kStreamRows / 2);
                if (n0 + 2 * unit + 1 < N)
                    C[static_cast<size_t>(row_at(p0 + t)) * ldc + n0 / 2 + unit] = from_f32<OutT>(stream_pair(act, sum(2 * unit, t), sum(2 * unit + 1, t), limit, alpha));
            }
        } else {
            for (int i = threadIdx.x; i < kStreamRows * rows; i += blockDim.x) {
                const int r = i % kStreamRows, t = i / kStreamRows;
                if (n0 + r >= N) continue;
                float v = sum(r, t);
                if (act == 1) {
                    v = fmaxf(v, 0.f);
                    v *= v;
                }
                C[static_cast<size_t>(row_at(p0 + t)) * ldc + n0 + r] = from_f32<OutT>(v);
            }
        }
    }
}

}  // namespace stride

using namespace stride;

extern "C" {

// C: [rows, N] (N / 2 with act 2 and 3), bfloat16 or float32. Returns -2 for what it does not take (K or lda no multiple of 8,
// unaligned operands, too many pairs); the caller then uses the other grouped product. ids null: rows by offsets and row_map;
// else pairs by ids [pairs], row p of A being pair p's token (top 1: the pair itself).
int stride_moe_stream(const void* A, int lda, const int32_t* row_map, const void* W, const int32_t* offsets, const int32_t* ids, int pairs, int top,
                      int experts, void* C, int ldc, int N, int K, int act, float limit, float alpha, const float* row_weight, int out_is_f32,
                      cudaStream_t stream) {
    if ((!ids && !offsets) || (ids && (pairs < 0 || top <= 0))) return STRIDE_BAD_ARGUMENT;
    if (ids && pairs > kStreamMaxPairs) return STRIDE_UNSUPPORTED;
    if (experts <= 0 || N <= 0 || K <= 0 || lda < K || act < 0 || act > 3 || ldc < (act >= 2 ? N / 2 : N) || (act >= 2 && N % 2)) return STRIDE_BAD_ARGUMENT;
    if (experts > 65535 || K % 8 || lda % 8 || (reinterpret_cast<uintptr_t>(A) | reinterpret_cast<uintptr_t>(W)) % 16) return STRIDE_UNSUPPORTED;
    const dim3 grid((N + kStreamRows - 1) / kStreamRows, experts), block(kStreamWarps * 32);
    if (out_is_f32)
        stride::launch(moe_stream_kernel<float>, grid, block, 0, stream, static_cast<const __nv_bfloat16*>(A), lda, row_map,
                       static_cast<const __nv_bfloat16*>(W), offsets, ids, pairs, top, static_cast<float*>(C), ldc, N, K, act, limit, alpha, row_weight);
    else
        stride::launch(moe_stream_kernel<__nv_bfloat16>, grid, block, 0, stream, static_cast<const __nv_bfloat16*>(A), lda, row_map,
                       static_cast<const __nv_bfloat16*>(W), offsets, ids, pairs, top, static_cast<__nv_bfloat16*>(C), ldc, N, K, act, limit, alpha, row_weight);
    return STRIDE_LAUNCH_STATUS();
}

}  // extern "C"

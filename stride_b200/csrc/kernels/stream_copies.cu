// A residual stream kept in n copies X_1 .. X_n per token (float32, a token's copies side by side: [tokens, n, width]).
// A sublayer reads a weighted sum of the copies and its output goes back to all of them at once
// (Zhu et al., "Hyper-Connections"):
//   write   X_b <- sum_a mix[a, b] X_a + out[b] * (scale . y)     every copy from the old ones; y the sublayer's output,
//                                                                 scale a learned vector over the width
//   read    u = sum_a in[a] X_a,  h = u / sqrt(mean(u^2) + eps) * w
// copies_step does the write behind one sublayer and the read in front of the next one in one pass over the copies, so they
// cross memory once a sublayer. Either half may be left out: no y (the first read), no norm (u itself is the result), no
// destination (the result is wanted for some rows only and the copies stay as they are). The source may hold one row a token
// instead of n (all copies equal, as the embedding leaves them): the first write spreads it out. `in` null: the plain sum.
// One CTA a token; float32 throughout; in float32 models the order of every sum depends on the row's sizes only.
#include "common.cuh"

namespace stride {

constexpr int kMaxCopies = 16;

struct CopiesArgs {
    const float* src;          // [tokens, n_src, width], n_src 1 or n
    float* dst;                // [tokens, n, width] or null; may be src when n_src == n
    const void* delta;         // [tokens, width] in the compute type, or null
    const float* scale;        // [width] or null
    const float* mix;          // [n, n], from-to
    const float* out_w;        // [n]
    const float* in_w;         // [n] or null
    const float* norm_w;       // [width] or null: no norm
    float eps;
    void* out;                 // [rows, width] in the compute type (norm_w given), or null
    float* sum_out;            // [rows, width] float32: u itself, or null
    const int32_t* rows;       // source row of every output row, or null
    int n_src, n, width;
};

template <typename T, int VEC>
__device__ __forceinline__ void load_compute(const T* p, float* v) {
    if constexpr (VEC == 1) {
        v[0] = to_f32(*p);
    } else if constexpr (sizeof(T) == 4) {
        const float4 r = *reinterpret_cast<const float4*>(p);
        v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
    } else {
        const uint2 r = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
        const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
        v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
    }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_compute(T* p, const float* v) {
    if constexpr (VEC == 1) {
        *p = from_f32<T>(v[0]);
    } else if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        uint2 r;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&r);
        h[0] = __floats2bfloat162_rn(v[0], v[1]);
        h[1] = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = r;
    }
}
template <int VEC>
__device__ __forceinline__ void load_float(const float* p, float* v) { load_compute<float, VEC>(p, v); }
template <int VEC>
__device__ __forceinline__ void store_float(float* p, const float* v) { store_compute<float, VEC>(p, v); }

// NS copies (NS 16: any number up to it, the rest weighted with zero); a thread handles packs of VEC columns: pack
// threadIdx.x + k * blockDim.x. The row's u waits in shared memory for the norm (every thread reads back only what it
// wrote). Up to four copies the coefficients sit in registers, beyond that they are read from shared memory.
template <typename T, int NS, int VEC>
__global__ void __launch_bounds__(512)
copies_step_kernel(const CopiesArgs p) {
    extern __shared__ __align__(16) float u_row[];        // width floats, when a norm is wanted
    __shared__ float scratch[32];
    constexpr bool IN_REGISTERS = NS <= 4;
    __shared__ float coef[IN_REGISTERS ? 1 : NS * NS + 2 * NS];       // mix, out, in
    const int n = NS <= 8 ? NS : p.n;
    pdl_trigger();
    // the coefficients are weights: no kernel writes them
    float reg[IN_REGISTERS ? NS * NS + 2 * NS : 1];
    auto from_memory = [&](int i) {
        const int a = i < NS * NS ? i / NS : i < NS * NS + NS ? i - NS * NS : i - NS * NS - NS, b = i < NS * NS ? i % NS : 0;
        if (a >= n || b >= n) return 0.f;
        if (i < NS * NS) return p.delta ? p.mix[a * n + b] : 0.f;
        if (i < NS * NS + NS) return p.delta ? p.out_w[a] : 0.f;
        return p.in_w ? p.in_w[a] : 1.f;
    };
    if constexpr (IN_REGISTERS) {
#pragma unroll
        for (int i = 0; i < NS * NS + 2 * NS; ++i) reg[i] = from_memory(i);
    } else {
        for (int i = threadIdx.x; i < NS * NS + 2 * NS; i += blockDim.x) coef[i] = from_memory(i);
        __syncthreads();
    }
    auto c = [&](int i) { return IN_REGISTERS ? reg[IN_REGISTERS ? i : 0] : coef[IN_REGISTERS ? 0 : i]; };
    auto mix = [&](int a, int b) { return c(a * NS + b); };
    auto ow = [&](int a) { return c(NS * NS + a); };
    auto iw = [&](int a) { return c(NS * NS + NS + a); };
    pdl_wait();
    const int r = blockIdx.x;
    const size_t t = p.rows ? static_cast<size_t>(p.rows[r]) : static_cast<size_t>(r);
    const int width = p.width;
    const float* src = p.src + t * p.n_src * width;
    float* dst = p.dst ? p.dst + t * n * width : nullptr;
    const T* delta = p.delta ? static_cast<const T*>(p.delta) + t * width : nullptr;
    float sq = 0.f;
    for (int i = threadIdx.x * VEC; i < width; i += blockDim.x * VEC) {
        float x[NS][VEC], u[VEC];
        if (p.n_src == 1) {
            load_float<VEC>(src + i, x[0]);
#pragma unroll
            for (int a = 1; a < NS; ++a)
#pragma unroll
                for (int e = 0; e < VEC; ++e) x[a][e] = x[0][e];
        } else {
#pragma unroll
            for (int a = 0; a < NS; ++a) {
                if (NS <= 8 || a < n) load_float<VEC>(src + static_cast<size_t>(a) * width + i, x[a]);
                else x[a][0] = 0.f;
            }
        }
        if (delta) {
            float y[VEC], s[VEC], nx[NS][VEC];
            load_compute<T, VEC>(delta + i, y);
            if (p.scale) {
                load_float<VEC>(p.scale + i, s);
#pragma unroll
                for (int e = 0; e < VEC; ++e) y[e] *= s[e];
            }
#pragma unroll
            for (int b = 0; b < NS; ++b)
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    float acc = ow(b) * y[e];
#pragma unroll
                    for (int a = 0; a < NS; ++a) acc = fmaf(mix(a, b), x[a][e], acc);
                    nx[b][e] = acc;
                }
#pragma unroll
            for (int a = 0; a < NS; ++a)
#pragma unroll
                for (int e = 0; e < VEC; ++e) x[a][e] = nx[a][e];
        }
        if (dst) {
#pragma unroll
            for (int a = 0; a < NS; ++a)
                if (NS <= 8 || a < n) store_float<VEC>(dst + static_cast<size_t>(a) * width + i, x[a]);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            u[e] = iw(0) * x[0][e];
#pragma unroll
            for (int a = 1; a < NS; ++a) u[e] = fmaf(iw(a), x[a][e], u[e]);
            sq = fmaf(u[e], u[e], sq);
        }
        if (p.sum_out) store_float<VEC>(p.sum_out + static_cast<size_t>(r) * width + i, u);
        if (p.norm_w) store_float<VEC>(u_row + i, u);
    }
    if (!p.norm_w) return;
    const float inv = rsqrtf(block_sum(sq, scratch) / static_cast<float>(width) + p.eps);
    T* out = static_cast<T*>(p.out) + static_cast<size_t>(r) * width;
    for (int i = threadIdx.x * VEC; i < width; i += blockDim.x * VEC) {
        float u[VEC], w[VEC];
        load_float<VEC>(u_row + i, u);
        load_float<VEC>(p.norm_w + i, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[e] = __fmul_rn(__fmul_rn(u[e], inv), w[e]);
        store_compute<T, VEC>(out + i, u);
    }
}

template <typename T, int NS, int VEC>
int launch_copies(const CopiesArgs& p, int num_rows, bool vec, cudaStream_t stream) {
    const int packs = vec ? p.width / 4 : p.width;
    int threads = (packs + 31) / 32 * 32;
    // many rows: small CTAs, several to an SM, keep more of the copies in flight (2,048 rows of 4 x 2,048: 26 us with 128 threads, 40 us
    // with 512); few rows: a row is worked through at once. In float32 the order of the norm's sum may not depend on the number of rows.
    const int limit = sizeof(T) == 4 ? 256 : num_rows >= 512 ? 128 : 512;
    threads = threads > limit ? limit : threads;
    const size_t smem = p.norm_w ? static_cast<size_t>(p.width) * sizeof(float) : 0;
    if (smem > 48 * 1024) {
        cudaError_t e = vec ? cudaFuncSetAttribute(copies_step_kernel<T, NS, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem))
                            : cudaFuncSetAttribute(copies_step_kernel<T, NS, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
        if (e != cudaSuccess) return static_cast<int>(e);
    }
    stride::launch(vec ? copies_step_kernel<T, NS, VEC> : copies_step_kernel<T, NS, 1>, dim3(num_rows), dim3(threads), smem, stream, p);
    return STRIDE_LAUNCH_STATUS();
}

template <typename T>
int dispatch_copies(const CopiesArgs& p, int n, int num_rows, bool vec, cudaStream_t stream) {
    switch (n) {
#define STRIDE_COPIES_CASE(N) case N: return launch_copies<T, N, 4>(p, num_rows, vec, stream);
        STRIDE_COPIES_CASE(1) STRIDE_COPIES_CASE(2) STRIDE_COPIES_CASE(3) STRIDE_COPIES_CASE(4)
        STRIDE_COPIES_CASE(5) STRIDE_COPIES_CASE(6) STRIDE_COPIES_CASE(7) STRIDE_COPIES_CASE(8)
#undef STRIDE_COPIES_CASE
        default: return n <= kMaxCopies ? launch_copies<T, kMaxCopies, 1>(p, num_rows, false, stream) : STRIDE_UNSUPPORTED;
    }
}

}  // namespace stride

using namespace stride;

// num_rows output rows (the step's tokens, or as many as `rows` names). dtype: that of delta and out.
extern "C" int stride_copies_step(const float* src, int n_src, float* dst, const void* delta, const float* scale, const float* mix,
                                  const float* out_w, const float* in_w, const float* norm_w, float eps, void* out, float* sum_out,
                                  const int32_t* rows, int num_rows, int n, int width, int dtype, cudaStream_t stream) {
    if (num_rows < 0 || n <= 0 || width <= 0 || !src || (n_src != 1 && n_src != n)) return STRIDE_BAD_ARGUMENT;
    if ((delta && (!mix || !out_w)) || (norm_w && !out) || (rows && dst) || (dst == src && n_src != n)) return STRIDE_BAD_ARGUMENT;
    if (n > kMaxCopies || width > 50000) return STRIDE_UNSUPPORTED;
    if (num_rows == 0) return 0;
    const CopiesArgs p = {src, dst, delta, scale, mix, out_w, in_w, norm_w, eps, out, sum_out, rows, n_src, n, width};
    auto aligned = [](const void* q) { return reinterpret_cast<uintptr_t>(q) % 16 == 0; };
    const bool vec = width % 4 == 0 && aligned(src) && aligned(dst) && aligned(delta) && aligned(scale) && aligned(norm_w) && aligned(out) &&
                     aligned(sum_out);
    if (dtype == STRIDE_DTYPE_F32) return dispatch_copies<float>(p, n, num_rows, vec, stream);
    if (dtype == STRIDE_DTYPE_BF16) return dispatch_copies<__nv_bfloat16>(p, n, num_rows, vec, stream);
    return STRIDE_BAD_ARGUMENT;
}

// The two maps of differential attention put together behind an attention kernel that treats them as heads of their own
// (pair_heads.cuh has the formula): x [tokens, 2 H, Dp] -> y [tokens, H, width].  One warp per (token, head), a lane's
// elements in rising order, then the warp's tree: a head's bits depend on nothing else.
#include "common.cuh"
#include "pair_heads.cuh"

#define PH_WARPS 8
#define PH_PER_LANE 16           // elements a lane keeps in registers: heads of up to 512

template <typename T, typename TO, int N>
__global__ void __launch_bounds__(32 * PH_WARPS)
pair_heads_kernel(const T* __restrict__ x, TO* __restrict__ y, PairOut p, long long heads, int Dp) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long h = (long long)blockIdx.x * PH_WARPS + (threadIdx.x >> 5);      // token * H + head
    if (h >= heads) return;
    const T* a = x + (size_t)h * 2 * Dp;
    const T* b = a + Dp;
    float o[N];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < N; i++) {
        const int d = i * 32 + lane;
        o[i] = d < p.vdim ? ld_f(a + d) - p.lam * ld_f(b + d) : 0.0f;
        ss += o[i] * o[i];
    }
    const float f = p.gain / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
    TO* dst = y + (size_t)h * p.width;
#pragma unroll
    for (int i = 0; i < N; i++) {
        const int d = i * 32 + lane;
        if (d < p.width) st_f(dst + d, o[i] * f);
    }
}

// rows of whole 16-byte pieces, float32 in and bfloat16 out: GROUP lanes (a power of two) per head, eight neighbouring
// elements per lane
template <int GROUP>
__global__ void __launch_bounds__(32 * PH_WARPS)
pair_heads8_kernel(const float* __restrict__ x, __nv_bfloat16* __restrict__ y, PairOut p, long long heads, int Dp) {
    pdl_trigger();
    pdl_wait();
    const int ln = threadIdx.x % GROUP, d = 8 * ln;
    const long long h = (long long)blockIdx.x * (32 * PH_WARPS / GROUP) + threadIdx.x / GROUP;
    const bool live = h < heads;                          // (no lane leaves before the shuffles)
    float o[8];
#pragma unroll
    for (int j = 0; j < 8; j++) o[j] = 0.0f;
    if (live && d < Dp) {
        const float4* pa = reinterpret_cast<const float4*>(x + (size_t)h * 2 * Dp + d);
        const float4* pb = reinterpret_cast<const float4*>(x + (size_t)h * 2 * Dp + Dp + d);
        const float4 a0 = pa[0], a1 = pa[1], b0 = pb[0], b1 = pb[1];
        const float fa[8] = {a0.x, a0.y, a0.z, a0.w, a1.x, a1.y, a1.z, a1.w}, fb[8] = {b0.x, b0.y, b0.z, b0.w, b1.x, b1.y, b1.z, b1.w};
#pragma unroll
        for (int j = 0; j < 8; j++) o[j] = d + j < p.vdim ? fa[j] - p.lam * fb[j] : 0.0f;
    }
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < 8; j++) ss += o[j] * o[j];
#pragma unroll
    for (int s = GROUP >> 1; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    const float f = p.gain / sqrtf(ss / (float)p.vdim + p.eps);
    if (live && d < p.width) {
        uint4 w;
        unsigned* wp = reinterpret_cast<unsigned*>(&w);
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const __nv_bfloat162 v = __floats2bfloat162_rn(o[2 * j] * f, o[2 * j + 1] * f);
            wp[j] = *reinterpret_cast<const unsigned*>(&v);
        }
        *reinterpret_cast<uint4*>(y + (size_t)h * p.width + d) = w;
    }
}

extern "C" int ri_pair_heads(const void* x, void* y, float lam, float eps, float gain, int tokens, int H, int Dp, int width,
                             int vdim, int dtype, int out_dtype, cudaStream_t stream) {
    // dtype: of x; out_dtype: of y (the same, or bfloat16 behind float32)
    if (tokens == 0) return 0;
    RI_REQUIRE(tokens > 0 && H > 0 && vdim > 0 && vdim <= Dp && vdim <= width, "pair_heads: bad sizes");
    RI_REQUIRE(width <= 32 * PH_PER_LANE, "pair_heads: rows of %d elements exceed the limit %d", width, 32 * PH_PER_LANE);
    const PairOut p{1, lam, eps, gain, vdim, width};
    const long long heads = (long long)tokens * H;
    if (dtype == RI_DTYPE_F32 && out_dtype == RI_DTYPE_BF16 && Dp % 8 == 0 && width % 8 == 0 && width <= Dp && Dp <= 256 && (((uintptr_t)x | (uintptr_t)y) & 15) == 0) {
        int group = 1;
        while (group < Dp / 8) group <<= 1;
        const int per = 32 * PH_WARPS / group;
        const dim3 grid((unsigned)((heads + per - 1) / per));
#define PH8(G)                                                                                                            \
    if (group == G)                                                                                                       \
        ri_launch_pdl(pair_heads8_kernel<G>, grid, dim3(32 * PH_WARPS), 0, stream, (const float*)x, (__nv_bfloat16*)y, \
                      p, heads, Dp)
        PH8(1);
        PH8(2);
        PH8(4);
        PH8(8);
        PH8(16);
        PH8(32);
#undef PH8
        RI_CHECK_LAUNCH("pair_heads");
        return 0;
    }
    const dim3 grid((unsigned)((heads + PH_WARPS - 1) / PH_WARPS));
#define PH_GO(T, TO)                                                                                                         \
    do {                                                                                                                     \
        if (width <= 128)                                                                                                    \
            ri_launch_pdl(pair_heads_kernel<T, TO, 4>, grid, dim3(32 * PH_WARPS), 0, stream, (const T*)x, (TO*)y, p, heads, Dp); \
        else                                                                                                                 \
            ri_launch_pdl(pair_heads_kernel<T, TO, PH_PER_LANE>, grid, dim3(32 * PH_WARPS), 0, stream, (const T*)x, (TO*)y, p, heads, Dp); \
    } while (0)
    if (dtype == RI_DTYPE_F32 && out_dtype == RI_DTYPE_F32) PH_GO(float, float);
    else if (dtype == RI_DTYPE_F32 && out_dtype == RI_DTYPE_BF16) PH_GO(float, __nv_bfloat16);
    else if (dtype == RI_DTYPE_BF16 && out_dtype == RI_DTYPE_BF16) PH_GO(__nv_bfloat16, __nv_bfloat16);
    else RI_FAIL(-1, "pair_heads: dtypes %d and %d", dtype, out_dtype);
#undef PH_GO
    RI_CHECK_LAUNCH("pair_heads");
    return 0;
}

// Dynamic Tanh in the place of a norm, and everything that happens to a row in front of it, element by element:
//     x' = x + float(y)                           (y: the output that the sublayer before left pending, or null)
//     out = tanh(alpha x') gain + bias            (alpha one number; gain, bias [dim] float32)
// x' is written back to the float32 residual unless only some rows are read.  There is no statistic over the row, so rows
// are cut into pieces as the launch likes and no result depends on the cut.  `embed_dyn_tanh` does the same to the rows of
// an embedding table: out = tanh(alpha (float(table[id]) scale)) gain + bias, in float32 (it is the residual itself).
// All arithmetic is float32 (tanhf); T is the compute type.
#include "common.cuh"
#include "linear_skinny_geometry.cuh"

#define DT_THREADS 256

__device__ __forceinline__ float4 dt_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 dt_ld4(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&u.x), b = *reinterpret_cast<const __nv_bfloat162*>(&u.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void dt_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void dt_st4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const unsigned*>(&a);
    u.y = *reinterpret_cast<const unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
}
__device__ __forceinline__ float dt_bend(float x, float alpha, float g, float b) { return fmaf(tanhf(alpha * x), g, b); }

struct DtArgs {
    float* resid;
    const void* y;
    const int* rows;
    const float *alpha, *gain, *bias;
    void* out;
    int n_rows, dim, pieces;           // a row is `pieces` blocks wide
    int hint_blocks;                   // blocks past the rows' ask for the weights that the linear after this norm reads first
    WeightHint next;
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(DT_THREADS) dyn_tanh_kernel(DtArgs a) {
    pdl_trigger();
    const int work = a.n_rows * a.pieces;
    if ((int)blockIdx.x >= work) {
        pdl_wait();
        weight_hint_prefetch(a.next, ((int)blockIdx.x - work) * DT_THREADS + (int)threadIdx.x, a.hint_blocks * DT_THREADS);
        return;
    }
    const int i = blockIdx.x / a.pieces, piece = blockIdx.x - i * a.pieces;
    const size_t r = a.rows ? (size_t)a.rows[i] : (size_t)i;
    const float alpha = a.alpha[0];
    const int e = (piece * DT_THREADS + (int)threadIdx.x) * (VEC ? 4 : 1);
    float* rp = a.resid + r * a.dim + e;
    T* op = (T*)a.out + (size_t)i * a.dim + e;
    const T* yp = a.y ? (const T*)a.y + r * a.dim + e : nullptr;
    if (VEC) {
        float4 g = make_float4(0.f, 0.f, 0.f, 0.f), b = g;
        if (e < a.dim) {
            g = dt_ld4(a.gain + e);
            b = dt_ld4(a.bias + e);
        }
        pdl_wait();
        if (e >= a.dim) return;
        float4 x = dt_ld4(rp);
        if (yp) {
            const float4 y = dt_ld4(yp);
            x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
            if (!a.rows) dt_st4(rp, x);
        }
        dt_st4(op, make_float4(dt_bend(x.x, alpha, g.x, b.x), dt_bend(x.y, alpha, g.y, b.y), dt_bend(x.z, alpha, g.z, b.z),
                               dt_bend(x.w, alpha, g.w, b.w)));
    } else {
        pdl_wait();
        if (e >= a.dim) return;
        float x = *rp;
        if (yp) {
            x += ld_f(yp);
            if (!a.rows) *rp = x;
        }
        st_f(op, dt_bend(x, alpha, a.gain[e], a.bias[e]));
    }
}

// resid [n, dim] float32; y [n, dim] of type `dtype` or null; rows: int32 indices of the rows to read (null: all n_rows, with
// write-back); out [n_rows, dim].  next_w [next_n, next_k] (bfloat16, or null): the weights of the weight-streaming linear
// that reads the result (a hint: it changes no result).
extern "C" int ri_dyn_tanh(float* resid, const void* y, const int* rows, const float* alpha, const float* gain,
                           const float* bias, void* out, int n_rows, int dim, int dtype, const void* next_w, int next_n,
                           int next_k, cudaStream_t stream) {
    if (n_rows == 0) return 0;
    RI_REQUIRE(n_rows > 0 && dim > 0, "dyn_tanh: bad sizes rows=%d dim=%d", n_rows, dim);
    RI_REQUIRE(dtype == RI_DTYPE_F32 || dtype == RI_DTYPE_BF16, "dyn_tanh: unknown dtype %d", dtype);
    const uintptr_t unit = dtype == RI_DTYPE_F32 ? 15 : 7;
    const bool vec = dim % 4 == 0 && (((uintptr_t)resid | (uintptr_t)gain | (uintptr_t)bias) & 15) == 0 &&
                     (((uintptr_t)y | (uintptr_t)out) & unit) == 0;
    DtArgs a;
    a.resid = resid; a.y = y; a.rows = rows; a.alpha = alpha; a.gain = gain; a.bias = bias; a.out = out;
    a.n_rows = n_rows; a.dim = dim;
    a.pieces = ((vec ? dim / 4 : dim) + DT_THREADS - 1) / DT_THREADS;
    a.next = make_weight_hint(nullptr, 0, 0, 0);
    a.hint_blocks = 0;
    if (next_w) {
        static int sms = 0;
        if (!sms) {
            int dev = 0;
            cudaGetDevice(&dev);
            cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
        }
        a.next = make_weight_hint(next_w, next_n, next_k, sms);
        if (a.next.base) {
            const long long lines = (long long)a.next.rows * SK_WARPS * (SK_HINT_STAGES * SK_STAGE_K * 2 / SK_HINT_LINE);
            const int want = (int)((lines + DT_THREADS * 2 - 1) / (DT_THREADS * 2));
            a.hint_blocks = want < 1 ? 1 : (want > 256 ? 256 : want);
        }
    }
    const long long blocks = (long long)n_rows * a.pieces + a.hint_blocks;
    RI_REQUIRE(blocks < (1ll << 31), "dyn_tanh: %d rows of %d elements: too many for one launch", n_rows, dim);
#define DT_GO(T, V) ri_launch_pdl(dyn_tanh_kernel<T, V>, dim3((unsigned)blocks), dim3(DT_THREADS), 0, stream, a)
    if (dtype == RI_DTYPE_F32) {
        if (vec) DT_GO(float, true); else DT_GO(float, false);
    } else {
        if (vec) DT_GO(__nv_bfloat16, true); else DT_GO(__nv_bfloat16, false);
    }
#undef DT_GO
    RI_CHECK_LAUNCH("dyn_tanh");
    return 0;
}

template <typename T>
__global__ void __launch_bounds__(DT_THREADS)
embed_dyn_tanh_kernel(const int* __restrict__ ids, const T* __restrict__ table, float scale, const float* __restrict__ alpha,
                      const float* __restrict__ gain, const float* __restrict__ bias, float* __restrict__ out, int dim, int vocab,
                      int vec, int* __restrict__ bad) {
    pdl_trigger();
    pdl_wait();
    const int id = ids[blockIdx.x];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0 && blockIdx.y == 0) atomicExch(bad, 1);
    const T* src = table + (size_t)(ok ? id : 0) * dim;
    float* dst = out + (size_t)blockIdx.x * dim;
    const float al = alpha[0];
    const int first = blockIdx.y * DT_THREADS + threadIdx.x, step = gridDim.y * DT_THREADS;
    if (vec) {
        for (int i = 4 * first; i < dim; i += 4 * step) {
            const float4 v = ok ? dt_ld4(src + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 g = dt_ld4(gain + i), b = dt_ld4(bias + i);
            dt_st4(dst + i, make_float4(dt_bend(v.x * scale, al, g.x, b.x), dt_bend(v.y * scale, al, g.y, b.y),
                                        dt_bend(v.z * scale, al, g.z, b.z), dt_bend(v.w * scale, al, g.w, b.w)));
        }
        return;
    }
    for (int i = first; i < dim; i += step) dst[i] = dt_bend((ok ? ld_f(src + i) : 0.0f) * scale, al, gain[i], bias[i]);
}

// out [tokens, dim] float32 from the rows of table [vocab, dim] (type `dtype`); an id outside the table is reported and its
// row taken as zeros
extern "C" int ri_embed_dyn_tanh(const int* ids, const void* table, float scale, const float* alpha, const float* gain,
                                 const float* bias, float* out, int tokens, int dim, int vocab, int dtype, int* bad_flag,
                                 cudaStream_t stream) {
    if (tokens == 0) return 0;
    RI_REQUIRE(tokens > 0 && dim > 0 && vocab > 0, "embed_dyn_tanh: bad sizes tokens=%d dim=%d vocab=%d", tokens, dim, vocab);
    const uintptr_t unit = dtype == RI_DTYPE_F32 ? 15 : 7;
    const int vec = dim % 4 == 0 && (((uintptr_t)gain | (uintptr_t)bias | (uintptr_t)out) & 15) == 0 && ((uintptr_t)table & unit) == 0;
    const int pieces = ((vec ? dim / 4 : dim) + DT_THREADS - 1) / DT_THREADS;
    const dim3 grid(tokens, pieces < 64 ? pieces : 64);
    if (dtype == RI_DTYPE_F32)
        ri_launch_pdl(embed_dyn_tanh_kernel<float>, grid, dim3(DT_THREADS), 0, stream, ids, (const float*)table, scale, alpha, gain,
                      bias, out, dim, vocab, vec, bad_flag);
    else if (dtype == RI_DTYPE_BF16)
        ri_launch_pdl(embed_dyn_tanh_kernel<__nv_bfloat16>, grid, dim3(DT_THREADS), 0, stream, ids, (const __nv_bfloat16*)table,
                      scale, alpha, gain, bias, out, dim, vocab, vec, bad_flag);
    else
        RI_FAIL(-1, "embed_dyn_tanh: unknown dtype %d", dtype);
    RI_CHECK_LAUNCH("embed_dyn_tanh");
    return 0;
}

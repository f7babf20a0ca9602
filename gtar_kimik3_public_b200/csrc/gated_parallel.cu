// Row-wise work of layers whose two branches read one stream through norms of their own (one number each) and are gated
// entry by entry, and the activation that norms three powers of a row.
//
//   gated_merge:  x += sigmoid(a_1 z_1 + b_1) * y_1 + sigmoid(a_2 z_2 + b_2) * y_2     (the second term may be absent)
//                 u = x / sqrt(mean(x^2) + eps) ;  n_1 = g_1 u ;  n_2 = g_2 u           (each only where it is asked for)
//                 z_1, z_2 lie side by side in one row; x is the 32-bit stream, updated in place.  Without branches the
//                 kernel only forms u, n_1 and n_2 of the stream.
//   poly_norm:    a N(z) + b N(z^2) + c N(z^3) + e,   N(y) = y / sqrt(mean(y^2) + eps), powers entry by entry
//
// One block per row with a fixed block size and all arithmetic in 32-bit: the order of a row's sums depends on nothing but
// the row's length.

#include "common.cuh"

namespace {

constexpr int ROW_THREADS = 256;

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// N consecutive entries as 32-bit numbers (N = 1: any address; N = 4: rows of whole 16- or 8-byte pieces)
template <int N, typename T>
__device__ __forceinline__ void load_n(const T* p, float (&v)[N]) {
    if constexpr (N == 1) {
        v[0] = to_float(*p);
    } else if constexpr (sizeof(T) == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
    } else {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v[0] = lo.x, v[1] = lo.y, v[2] = hi.x, v[3] = hi.y;
    }
}
template <int N, typename T>
__device__ __forceinline__ void store_n(T* p, const float (&v)[N]) {
    if constexpr (N == 1) {
        *p = from_float<T>(v[0]);
    } else if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<uint32_t*>(&lo);
        raw.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = raw;
    }
}

struct MergeGates {
    const float* bias_1;
    const float* bias_2;
    float gain_1, gain_2;
};

template <typename T, typename T2, int N>
__global__ void __launch_bounds__(ROW_THREADS) gated_merge_kernel(
    float* __restrict__ x, const T* __restrict__ z, long long ld_z, const T* __restrict__ y_1, const T2* __restrict__ y_2,
    MergeGates gates, T* __restrict__ u, T* __restrict__ n_1, T* __restrict__ n_2, float next_gain_1, float next_gain_2, float eps,
    int width) {
    extern __shared__ __align__(16) float row[];  // width floats
    __shared__ float scratch[33];
    pdl_launch_dependents();
    const size_t at = (size_t)blockIdx.x * width;
    pdl_wait();
    float ss = 0.f;
    for (int i = threadIdx.x * N; i < width; i += ROW_THREADS * N) {
        float v[N];
        load_n<N>(x + at + i, v);
        if (y_1 != nullptr) {
            float zz[N], y[N], b[N];
            load_n<N>(z + (size_t)blockIdx.x * ld_z + i, zz);
            load_n<N>(y_1 + at + i, y);
            load_n<N>(gates.bias_1 + i, b);
            float add[N];
#pragma unroll
            for (int e = 0; e < N; ++e) add[e] = sigmoid_f(fmaf(gates.gain_1, zz[e], b[e])) * y[e];
            if (y_2 != nullptr) {
                load_n<N>(z + (size_t)blockIdx.x * ld_z + width + i, zz);
                load_n<N>(y_2 + at + i, y);
                load_n<N>(gates.bias_2 + i, b);
#pragma unroll
                for (int e = 0; e < N; ++e) add[e] = fmaf(sigmoid_f(fmaf(gates.gain_2, zz[e], b[e])), y[e], add[e]);
            }
#pragma unroll
            for (int e = 0; e < N; ++e) v[e] += add[e];
            store_n<N>(x + at + i, v);
        }
        if (u != nullptr) {
            store_n<N>(row + i, v);
#pragma unroll
            for (int e = 0; e < N; ++e) ss = fmaf(v[e], v[e], ss);
        }
    }
    if (u == nullptr) return;
    ss = block_sum(ss, scratch);
    const float r = 1.f / sqrtf(ss / (float)width + eps);
    for (int i = threadIdx.x * N; i < width; i += ROW_THREADS * N) {  // each thread reads back what it wrote itself
        float v[N], o[N];
        load_n<N>(row + i, v);
#pragma unroll
        for (int e = 0; e < N; ++e) v[e] *= r;
        store_n<N>(u + at + i, v);
#pragma unroll
        for (int e = 0; e < N; ++e) o[e] = v[e] * next_gain_1;
        store_n<N>(n_1 + at + i, o);
        if (n_2 != nullptr) {
#pragma unroll
            for (int e = 0; e < N; ++e) o[e] = v[e] * next_gain_2;
            store_n<N>(n_2 + at + i, o);
        }
    }
}

// Sums of three numbers over the block, every thread gets them.  `scratch` holds 3 * (ROW_THREADS / 32) floats.
__device__ __forceinline__ void block_sum3(float (&v)[3], float* scratch) {
    constexpr int WARPS = ROW_THREADS / 32;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
    for (int c = 0; c < 3; ++c) {
        const float s = warp_sum(v[c]);
        if (lane == 0) scratch[c * WARPS + warp] = s;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 3; ++c) {
        float s = 0.f;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) s += scratch[c * WARPS + w];
        v[c] = s;
    }
}

template <typename TI, typename TO, int N>
__global__ void __launch_bounds__(ROW_THREADS) poly_norm_kernel(const TI* __restrict__ z, TO* __restrict__ out, int width, float a,
                                                                float b, float c, float e, float eps) {
    extern __shared__ __align__(16) float row[];  // width floats
    __shared__ float scratch[3 * (ROW_THREADS / 32)];
    pdl_launch_dependents();
    pdl_wait();
    const size_t at = (size_t)blockIdx.x * width;
    float sums[3] = {0.f, 0.f, 0.f};  // of z^2, z^4, z^6
    for (int i = threadIdx.x * N; i < width; i += ROW_THREADS * N) {
        float v[N];
        load_n<N>(z + at + i, v);
        store_n<N>(row + i, v);
#pragma unroll
        for (int k = 0; k < N; ++k) {
            const float s = v[k] * v[k], q = s * s;
            sums[0] += s;
            sums[1] += q;
            sums[2] = fmaf(q, s, sums[2]);
        }
    }
    block_sum3(sums, scratch);
    const float n = (float)width;
    const float ra = a / sqrtf(sums[0] / n + eps), rb = b / sqrtf(sums[1] / n + eps), rc = c / sqrtf(sums[2] / n + eps);
    for (int i = threadIdx.x * N; i < width; i += ROW_THREADS * N) {  // each thread reads back what it wrote itself
        float v[N];
        load_n<N>(row + i, v);
#pragma unroll
        for (int k = 0; k < N; ++k) {
            const float w = v[k], s = w * w;
            v[k] = fmaf(rc, s * w, fmaf(rb, s, fmaf(ra, w, e)));
        }
        store_n<N>(out + at + i, v);
    }
}

bool aligned(const void* p, int bytes) { return p == nullptr || reinterpret_cast<uintptr_t>(p) % bytes == 0; }

}  // namespace

// dtype: of z, y_1 and the outputs; y2_dtype: of y_2.  y_1 null: no branches.  u null: no norms.  n_1 goes with u; n_2 may be null.
GK_EXPORT int gk_gated_merge(float* x, int dtype, const void* z, long long ld_z, const void* y_1, const void* y_2, int y2_dtype,
                             const float* bias_1, const float* bias_2, float gain_1, float gain_2, void* u, void* n_1, void* n_2,
                             float next_gain_1, float next_gain_2, float eps, int rows, int width, void* stream) {
    GK_REQUIRE(GK_VALID_DTYPE(dtype) && GK_VALID_DTYPE(y2_dtype), "gated_merge: bad dtype");
    GK_REQUIRE(rows >= 0 && width > 0, "gated_merge: bad sizes");
    GK_REQUIRE(y_1 != nullptr ? (z != nullptr && bias_1 != nullptr && ld_z >= (y_2 != nullptr ? 2 : 1) * (long long)width) : y_2 == nullptr,
               "gated_merge: a branch needs its gate");
    GK_REQUIRE(y_2 == nullptr || bias_2 != nullptr, "gated_merge: the second branch needs its gate");
    GK_REQUIRE(u == nullptr ? (n_1 == nullptr && n_2 == nullptr) : (n_1 != nullptr && eps > 0.f), "gated_merge: the norms come together");
    GK_REQUIRE((size_t)width * sizeof(float) <= 200 * 1024, "gated_merge: rows of %d are longer than the kernel stages", width);
    if (rows == 0) return GK_OK;
    const MergeGates gates = {bias_1, bias_2, gain_1, gain_2};
    const bool vec = width % 4 == 0 && ld_z % 4 == 0 && aligned(x, 16) && aligned(z, 16) && aligned(y_1, 16) && aligned(y_2, 16) &&
                     aligned(bias_1, 16) && aligned(bias_2, 16) && aligned(u, 16) && aligned(n_1, 16) && aligned(n_2, 16);
    const size_t smem = (size_t)width * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
#define GK_MERGE(N)                                                                                                                  \
    do {                                                                                                                             \
        if (smem > 48 * 1024)                                                                                                        \
            cudaFuncSetAttribute(gated_merge_kernel<T, T2, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);             \
        gk_launch(gated_merge_kernel<T, T2, N>, dim3(rows), dim3(ROW_THREADS), smem, s, x, (const T*)z, ld_z, (const T*)y_1,         \
                  (const T2*)y_2, gates, (T*)u, (T*)n_1, (T*)n_2, next_gain_1, next_gain_2, eps, width);                             \
    } while (0)
    GK_DISPATCH_DTYPE(dtype, T, {
        GK_DISPATCH_DTYPE(y2_dtype, T2, {
            if (vec) GK_MERGE(4);
            else GK_MERGE(1);
        })
    })
#undef GK_MERGE
    GK_CHECK_LAUNCH("gated_merge");
    return GK_OK;
}

GK_EXPORT int gk_poly_norm(const void* z, int z_dtype, void* out, int out_dtype, int rows, int width, float a, float b, float c, float e,
                           float eps, void* stream) {
    GK_REQUIRE(GK_VALID_DTYPE(z_dtype) && GK_VALID_DTYPE(out_dtype), "poly_norm: bad dtype");
    GK_REQUIRE(rows >= 0 && width > 0 && eps > 0.f, "poly_norm: bad sizes");
    GK_REQUIRE((size_t)width * sizeof(float) <= 200 * 1024, "poly_norm: rows of %d are longer than the kernel stages", width);
    if (rows == 0) return GK_OK;
    const bool vec = width % 4 == 0 && aligned(z, 16) && aligned(out, 16);
    const size_t smem = (size_t)width * sizeof(float);
    cudaStream_t s = (cudaStream_t)stream;
#define GK_POLY(N)                                                                                                                   \
    do {                                                                                                                             \
        if (smem > 48 * 1024)                                                                                                        \
            cudaFuncSetAttribute(poly_norm_kernel<TI, TO, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);              \
        gk_launch(poly_norm_kernel<TI, TO, N>, dim3(rows), dim3(ROW_THREADS), smem, s, (const TI*)z, (TO*)out, width, a, b, c, e, eps); \
    } while (0)
    GK_DISPATCH_DTYPE(z_dtype, TI, {
        GK_DISPATCH_DTYPE(out_dtype, TO, {
            if (vec) GK_POLY(4);
            else GK_POLY(1);
        })
    })
#undef GK_POLY
    GK_CHECK_LAUNCH("poly_norm");
    return GK_OK;
}

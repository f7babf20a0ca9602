// The gated delta rule with ONE decay per head: what stands between its packed input projection and its output projection.
//
// Per sequence and head, with a state S [d, dv] of 32-bit floats that starts at zero:
//     S <- g_t S ;  u_t = beta_t (v_t - S^T k_t) ;  S <- S + k_t u_t^T ;  o_t = S^T q_t
// where q_t, k_t come out of a short causal convolution over time and SiLU and are scaled to unit length per
// head (q also by d^-1/2), v_t out of a convolution and SiLU, beta_t = sigmoid(b_t) and
// g_t = exp(-exp(A_h) * softplus(a_t + dt_bias_h)).  A head's read-out is divided by its root mean square, multiplied by a
// weight shared by the heads and by silu(gate).
//
// The projection holds, from a column that the caller names, q (G d) | k (G d) | v (H dv) | b (H) | a (H) | gate (H dv).
// A sequence's convolution state is a ring of `taps` rows: the input at position p lies in row p % taps.  A step that
// reads the taps - 1 inputs before its own never touches the row it writes, so blocks that share an input need no order
// among them.
//
//   delta_head_prepare  many tokens: a warp per (unit, some consecutive tokens), units being the heads of q, of k and of v.  The
//                       convolution's window slides in registers, so that an input is fetched once for its tokens.  The
//                       results are either 32-bit vectors (what the token-by-token recurrence reads: unit lengths done,
//                       decays as factors) or, for the chunked recurrence, the activations rounded to bfloat16 with a
//                       32-bit factor per head beside them that makes the rounded vector a unit vector, and the decays'
//                       logarithms.
//   conv_ring           leaves the step's last inputs in the sequences' rings (after every reader of the old rows is done)
//   delta_head_single   steps of one token a sequence, everything above in one kernel: a block per sequence and head holds the
//                       head's state in registers, 4 columns and up to 16 rows a thread, fetched once and stored once.

#include "common.cuh"

namespace {

constexpr int PREP_WARPS = 4;
constexpr int MAX_TAPS = 16;

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// with the hardware's exponential and division, where the result is rounded to bfloat16
__device__ __forceinline__ float silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }

struct HeadSizes {
    int n_heads, n_kv, d, dv, taps;
    __device__ __forceinline__ int qk() const { return n_kv * d; }
    __device__ __forceinline__ int channels() const { return 2 * n_kv * d + n_heads * dv; }
    __device__ __forceinline__ int b_at() const { return channels(); }
    __device__ __forceinline__ int a_at() const { return channels() + n_heads; }
    __device__ __forceinline__ int gate_at() const { return channels() + 2 * n_heads; }
};

template <typename T, int VEC>
__device__ __forceinline__ void load_vec(const T* p, float (&v)[VEC]) {
    if constexpr (VEC == 4 && sizeof(T) == 4) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w;
    } else if constexpr (VEC == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v[0] = lo.x, v[1] = lo.y, v[2] = hi.x, v[3] = hi.y;
    } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = to_float(p[e]);
    }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[VEC]) {
    if constexpr (VEC == 4 && sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else if constexpr (VEC == 4) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        uint2 raw;
        raw.x = *reinterpret_cast<uint32_t*>(&lo);
        raw.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = raw;
    } else {
#pragma unroll
        for (int e = 0; e < VEC; ++e) p[e] = from_float<T>(v[e]);
    }
}

// The outputs: 32-bit (TO float): q, k unit vectors, v, g the decay factors.  bfloat16 (TO bfloat16): the rounded
// activations, with q_unit, k_unit [T, G] and g the decays' logarithms.
template <typename TO>
struct PrepareOut {
    TO *q, *k, *v;
    float *q_unit, *k_unit, *g, *beta;
};

// TAPS: the number of taps, or 0 for any (the window then comes from memory tap by tap).  E: pieces of 32 VEC channels a head.
template <typename T, typename TO, int VEC, int TAPS, int E>
__global__ void __launch_bounds__(PREP_WARPS * 32) delta_head_prepare_kernel(
    const T* __restrict__ proj, long long ld, const float* __restrict__ conv_w /* [taps, C] */,
    const float* __restrict__ ring /* [slots, taps, C] */, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
    const int* __restrict__ tok_pos, const int* __restrict__ tok_seq, const int* __restrict__ cu_q, const int* __restrict__ slots,
    PrepareOut<TO> out, int n_tokens, HeadSizes sz, int per_warp) {
    constexpr bool ROUNDED = sizeof(TO) == 2;
    constexpr int WINDOW = TAPS > 1 ? TAPS - 1 : 1;
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, units = 2 * sz.n_kv + sz.n_heads;
    const int strips = (n_tokens + per_warp - 1) / per_warp;
    const long long item = (long long)blockIdx.x * PREP_WARPS + (threadIdx.x >> 5);
    if (item >= (long long)strips * units) return;
    const int strip = (int)(item / units), unit = (int)(item - (long long)strip * units);
    const int t_begin = strip * per_warp, t_end = min(n_tokens, t_begin + per_warp);
    const int taps = TAPS > 0 ? TAPS : sz.taps, C = sz.channels();
    const bool is_qk = unit < 2 * sz.n_kv, is_q = unit < sz.n_kv;
    const int h = unit - 2 * sz.n_kv;
    const int width = is_qk ? sz.d : sz.dv;
    const int c0 = is_qk ? unit * sz.d : 2 * sz.qk() + h * sz.dv;
    float w[TAPS > 0 ? TAPS : 1][E][VEC], past[WINDOW][E][VEC];  // past[j - 1]: the input j tokens back
    if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j)
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const int i = (e * 32 + lane) * VEC;
                if (i < width) load_vec<float, VEC>(conv_w + (size_t)j * C + c0 + i, w[j][e]);
            }
    }
    const float scale = 1.f / sqrtf((float)sz.d);
    const float rate = is_qk ? 0.f : -expf(a_log[h]);
    const float dt = is_qk ? 0.f : dt_bias[h];
    for (int t = t_begin; t < t_end; ++t) {
        const int seq = tok_seq[t], in_step = t - cu_q[seq];
        const bool fresh = TAPS > 1 && (t == t_begin || in_step == 0);
        const int pos = tok_pos[t];
        const float* mine = ring + (size_t)slots[seq] * taps * C + c0;
        auto earlier = [&](int j, int i, float (&v)[VEC]) {  // the input j tokens back
            if (in_step >= j) load_vec<T, VEC>(proj + (size_t)(t - j) * ld + c0 + i, v);
            else if (pos >= j) load_vec<float, VEC>(mine + (size_t)((pos - j) % taps) * C + i, v);
            else {
#pragma unroll
                for (int x = 0; x < VEC; ++x) v[x] = 0.f;
            }
        };
        float act[E][VEC], ss = 0.f;
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int i = (e * 32 + lane) * VEC;
#pragma unroll
            for (int x = 0; x < VEC; ++x) act[e][x] = 0.f;
            if (i >= width) continue;
            float own[VEC];
            load_vec<T, VEC>(proj + (size_t)t * ld + c0 + i, own);
            // a token's sum takes the taps from the current token's backward, whatever the path
            if constexpr (TAPS > 0) {
                if constexpr (TAPS > 1) {
                    if (fresh) {
#pragma unroll
                        for (int j = 1; j < TAPS; ++j) earlier(j, i, past[j - 1][e]);
                    }
                }
#pragma unroll
                for (int x = 0; x < VEC; ++x) {
                    float y = w[TAPS - 1][e][x] * own[x];
#pragma unroll
                    for (int j = 1; j < TAPS; ++j) y = fmaf(w[TAPS - 1 - j][e][x], past[j - 1][e][x], y);
                    act[e][x] = ROUNDED ? silu_fast(y) : silu_f(y);
                }
                if constexpr (TAPS > 1) {
#pragma unroll
                    for (int x = 0; x < VEC; ++x) {
#pragma unroll
                        for (int j = TAPS - 1; j > 1; --j) past[j - 1][e][x] = past[j - 2][e][x];
                        past[0][e][x] = own[x];
                    }
                }
            } else {
                float y[VEC], wj[VEC], v[VEC];
                load_vec<float, VEC>(conv_w + (size_t)(taps - 1) * C + c0 + i, wj);
#pragma unroll
                for (int x = 0; x < VEC; ++x) y[x] = wj[x] * own[x];
                for (int j = 1; j < taps; ++j) {
                    load_vec<float, VEC>(conv_w + (size_t)(taps - 1 - j) * C + c0 + i, wj);
                    earlier(j, i, v);
#pragma unroll
                    for (int x = 0; x < VEC; ++x) y[x] = fmaf(wj[x], v[x], y[x]);
                }
#pragma unroll
                for (int x = 0; x < VEC; ++x) act[e][x] = ROUNDED ? silu_fast(y[x]) : silu_f(y[x]);
            }
            if (is_qk) {
#pragma unroll
                for (int x = 0; x < VEC; ++x) {
                    if (ROUNDED) act[e][x] = to_float(from_float<TO>(act[e][x]));
                    ss = fmaf(act[e][x], act[e][x], ss);
                }
            }
        }
        TO* dst;
        if (is_qk) {
            ss = warp_sum(ss);
            float r = 1.f / sqrtf(ss + 1e-6f);
            if (is_q) r *= scale;
            const int a = is_q ? unit : unit - sz.n_kv;
            dst = (is_q ? out.q : out.k) + ((size_t)t * sz.n_kv + a) * sz.d;
            if (ROUNDED) {
                if (lane == 0) (is_q ? out.q_unit : out.k_unit)[(size_t)t * sz.n_kv + a] = r;
            } else {
#pragma unroll
                for (int e = 0; e < E; ++e)
#pragma unroll
                    for (int x = 0; x < VEC; ++x) act[e][x] *= r;
            }
        } else {
            dst = out.v + ((size_t)t * sz.n_heads + h) * sz.dv;
            if (lane == 0) {
                const T* row = proj + (size_t)t * ld;
                const float log_g = rate * softplus_f(to_float(row[sz.a_at() + h]) + dt);
                out.g[(size_t)t * sz.n_heads + h] = ROUNDED ? log_g : expf(log_g);
                out.beta[(size_t)t * sz.n_heads + h] = sigmoid_f(to_float(row[sz.b_at() + h]));
            }
        }
#pragma unroll
        for (int e = 0; e < E; ++e) {
            const int i = (e * 32 + lane) * VEC;
            if (i < width) store_vec<TO, VEC>(dst + i, act[e]);
        }
    }
}

// A thread per (sequence, channel): the step's last inputs go to the rows of their positions.
template <typename T>
__global__ void conv_ring_kernel(const T* __restrict__ proj, long long ld, float* __restrict__ ring, const int* __restrict__ cu_q,
                                 const int* __restrict__ kv_len, const int* __restrict__ slots, int C, int taps) {
    pdl_launch_dependents();
    pdl_wait();
    const int seq = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= C) return;
    const int end = cu_q[seq + 1], n = end - cu_q[seq], last = kv_len[seq] - 1;
    float* mine = ring + (size_t)slots[seq] * taps * C + c;
    for (int j = 0; j < min(n, taps - 1); ++j) mine[(size_t)((last - j) % taps) * C] = to_float(proj[(size_t)(end - 1 - j) * ld + c]);
}

// One token a sequence.  A block per (head, sequence); NT threads as CG groups of 4 columns by NT / CG groups of rows, R rows
// a thread.  Sums over the rows meet in shared memory in the order of the row groups.
// TAPS: 4, or 0 for any number of taps.
template <typename T, int NT, int CG, int R, int TAPS>
__global__ void __launch_bounds__(NT) delta_head_single_kernel(
    const T* __restrict__ proj, long long ld, const float* __restrict__ conv_w, float* ring, const float* __restrict__ a_log,
    const float* __restrict__ dt_bias, const float* __restrict__ norm_w, float* __restrict__ state /* [slots, H, d, dv] */,
    const int* __restrict__ tok_pos, const int* __restrict__ tok_seq, const int* __restrict__ slots, T* __restrict__ out,
    long long ld_out, float out_scale, float eps, HeadSizes sz) {
    constexpr int RG = NT / CG;
    extern __shared__ __align__(16) float smem[];
    const int d = sz.d, dv = sz.dv, taps = sz.taps, C = sz.channels();
    const int d4 = (d + 3) & ~3, dv4 = (dv + 3) & ~3;
    float* sq = smem;                 // [d4]
    float* sk = sq + d4;              // [d4]
    float* sv = sk + d4;              // [dv4]
    float* so = sv + dv4;             // [dv4]
    float* part = so + dv4;           // [RG][2][CG * 4]
    pdl_launch_dependents();
    const int head = blockIdx.x, t = blockIdx.y;
    const int group = sz.n_heads / sz.n_kv, hk = head / group;
    const int cg = threadIdx.x % CG, rg = threadIdx.x / CG, lane = threadIdx.x & 31;
    const bool live = cg * 4 < dv;
    // the channels of the head's q, k and v: at most three a thread
    constexpr int TURNS = 3;
    auto channel = [&](int i) { return i < d ? hk * d + i : i < 2 * d ? sz.qk() + hk * d + (i - d) : 2 * sz.qk() + head * dv + (i - 2 * d); };
    float w[TURNS][TAPS > 0 ? TAPS : 1];
    if constexpr (TAPS > 0) {  // no kernel in flight writes the weights
#pragma unroll
        for (int n = 0; n < TURNS; ++n) {
            const int i = n * NT + threadIdx.x;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[n][j] = i < 2 * d + dv ? conv_w[(size_t)(TAPS - 1 - j) * C + channel(i)] : 0.f;
        }
    }
    pdl_wait();
    const size_t slot = (size_t)slots[tok_seq[t]];
    const int pos = tok_pos[t];
    float* mine = state + (slot * sz.n_heads + head) * (size_t)d * dv + cg * 4;
    float S[R][4];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int row = r * RG + rg;
#pragma unroll
        for (int x = 0; x < 4; ++x) S[r][x] = 0.f;
        if (live && row < d) load_vec<float, 4>(mine + (size_t)row * dv, S[r]);
    }
    const T* row_t = proj + (size_t)t * ld;
    const T* gate = row_t + sz.gate_at() + (size_t)head * dv;
    const float my_gate = (int)threadIdx.x < dv ? to_float(gate[threadIdx.x]) : 0.f;  // dv <= NT
    const float my_weight = (int)threadIdx.x < dv ? norm_w[threadIdx.x] : 0.f;
    const float beta = sigmoid_f(to_float(row_t[sz.b_at() + head]));
    const float g = expf(-expf(a_log[head]) * softplus_f(to_float(row_t[sz.a_at() + head]) + dt_bias[head]));
    // the convolutions of the head's q, k and v; the first head of a group leaves q's and k's inputs in the ring
    float* ring_rows = ring + slot * taps * C;
    const bool owner = head % group == 0;
    if constexpr (TAPS > 0) {
        float x[TURNS][TAPS];  // all inputs on their way before the first store to the ring
#pragma unroll
        for (int n = 0; n < TURNS; ++n) {
            const int i = n * NT + threadIdx.x;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                x[n][j] = 0.f;
                if (i < 2 * d + dv) {
                    if (j == 0) x[n][j] = to_float(row_t[channel(i)]);
                    else if (j <= pos) x[n][j] = ring_rows[(size_t)((pos - j) % TAPS) * C + channel(i)];
                }
            }
        }
#pragma unroll
        for (int n = 0; n < TURNS; ++n) {
            const int i = n * NT + threadIdx.x;
            if (i >= 2 * d + dv) continue;
            float y = w[n][0] * x[n][0];
#pragma unroll
            for (int j = 1; j < TAPS; ++j) y = fmaf(w[n][j], x[n][j], y);
            if (TAPS > 1 && (owner || i >= 2 * d)) ring_rows[(size_t)(pos % TAPS) * C + channel(i)] = x[n][0];
            (i < d ? sq[i] : i < 2 * d ? sk[i - d] : sv[i - 2 * d]) = silu_f(y);
        }
    } else {
        for (int i = threadIdx.x; i < 2 * d + dv; i += NT) {
            const int c = channel(i);
            const float own = to_float(row_t[c]);
            float y = conv_w[(size_t)(taps - 1) * C + c] * own;
            for (int j = 1; j < taps && j <= pos; ++j) y = fmaf(conv_w[(size_t)(taps - 1 - j) * C + c], ring_rows[(size_t)((pos - j) % taps) * C + c], y);
            if (taps > 1 && (owner || i >= 2 * d)) ring_rows[(size_t)(pos % taps) * C + c] = own;
            (i < d ? sq[i] : i < 2 * d ? sk[i - d] : sv[i - 2 * d]) = silu_f(y);
        }
    }
    __syncthreads();
    float qq = 0.f, kk = 0.f, qk = 0.f;  // every warp forms the three sums for itself
    for (int i = lane; i < d; i += 32) {
        qq = fmaf(sq[i], sq[i], qq);
        kk = fmaf(sk[i], sk[i], kk);
        qk = fmaf(sq[i], sk[i], qk);
    }
    qq = warp_sum(qq), kk = warp_sum(kk), qk = warp_sum(qk);
    const float rk = 1.f / sqrtf(kk + 1e-6f), rq = 1.f / sqrtf(qq + 1e-6f) * (1.f / sqrtf((float)d));
    float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int row = r * RG + rg;
        const float kr = row < d ? sk[row] * rk : 0.f, qr = row < d ? sq[row] * rq : 0.f;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            S[r][x] *= g;
            a[x] = fmaf(S[r][x], kr, a[x]);
            b[x] = fmaf(S[r][x], qr, b[x]);
        }
    }
    *reinterpret_cast<float4*>(part + ((size_t)rg * 2) * CG * 4 + cg * 4) = make_float4(a[0], a[1], a[2], a[3]);
    *reinterpret_cast<float4*>(part + ((size_t)rg * 2 + 1) * CG * 4 + cg * 4) = make_float4(b[0], b[1], b[2], b[3]);
    __syncthreads();
    float u[4] = {0.f, 0.f, 0.f, 0.f};
    for (int i = 0; i < RG; ++i) {
        const float4 p = *reinterpret_cast<const float4*>(part + ((size_t)i * 2) * CG * 4 + cg * 4);
        u[0] += p.x, u[1] += p.y, u[2] += p.z, u[3] += p.w;
    }
    if (live) {
#pragma unroll
        for (int x = 0; x < 4; ++x) u[x] = beta * (sv[cg * 4 + x] - u[x]);
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int row = r * RG + rg;
            if (row >= d) continue;
            const float kr = sk[row] * rk;
#pragma unroll
            for (int x = 0; x < 4; ++x) S[r][x] = fmaf(kr, u[x], S[r][x]);
            store_vec<float, 4>(mine + (size_t)row * dv, S[r]);
        }
        if (rg == 0) {  // o = (g S)^T q + (k . q) u
            float o[4] = {0.f, 0.f, 0.f, 0.f};
            for (int i = 0; i < RG; ++i) {
                const float4 p = *reinterpret_cast<const float4*>(part + ((size_t)i * 2 + 1) * CG * 4 + cg * 4);
                o[0] += p.x, o[1] += p.y, o[2] += p.z, o[3] += p.w;
            }
            const float c = qk * rq * rk;
#pragma unroll
            for (int x = 0; x < 4; ++x) so[cg * 4 + x] = fmaf(c, u[x], o[x]);
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int i = lane; i < dv; i += 32) ss = fmaf(so[i], so[i], ss);
    ss = warp_sum(ss);
    const float r = out_scale / sqrtf(ss / (float)dv + eps);
    if ((int)threadIdx.x < dv)
        out[(size_t)t * ld_out + (size_t)head * dv + threadIdx.x] = from_float<T>(so[threadIdx.x] * r * my_weight * silu_f(my_gate));
}

bool sizes_ok(int n_heads, int n_kv, int d, int dv, int taps) {
    return n_heads > 0 && n_kv > 0 && n_heads % n_kv == 0 && d > 0 && dv > 0 && taps >= 1 && taps <= MAX_TAPS;
}

template <typename T, typename TO, int VEC, int TAPS>
int prepare_as(const void* proj, long long ld, const float* conv_w, const float* ring, const float* a_log, const float* dt_bias,
               const int* tok_pos, const int* tok_seq, const int* cu_q, const int* slots, PrepareOut<TO> out, int n_tokens, HeadSizes sz,
               cudaStream_t s) {
    const int widest = sz.d > sz.dv ? sz.d : sz.dv;
    const int pieces = (widest + 32 * VEC - 1) / (32 * VEC);
    const int units = 2 * sz.n_kv + sz.n_heads;
    // few tokens: one a warp; many: strips, so that an input is fetched once for several tokens
    int per_warp = 1;
    while (per_warp < 8 && (long long)n_tokens * units / (per_warp * 2) >= 2368) per_warp *= 2;
    const long long items = (long long)((n_tokens + per_warp - 1) / per_warp) * units;
    const long long blocks = (items + PREP_WARPS - 1) / PREP_WARPS;
    GK_REQUIRE(blocks < 2147483647LL, "delta_head_prepare: too many tokens");
#define GK_PREPARE(E)                                                                                                                  \
    gk_launch(delta_head_prepare_kernel<T, TO, VEC, TAPS, E>, dim3((unsigned)blocks), dim3(PREP_WARPS * 32), 0, s, (const T*)proj, ld, \
              conv_w, ring, a_log, dt_bias, tok_pos, tok_seq, cu_q, slots, out, n_tokens, sz, per_warp)
    if (pieces <= 1) GK_PREPARE(1);
    else if (pieces <= 2) GK_PREPARE(2);
    else if (VEC == 4 || pieces <= 4) GK_PREPARE(4);  // heads have at most 512 entries
    else GK_PREPARE(VEC == 4 ? 4 : 16);
#undef GK_PREPARE
    GK_CHECK_LAUNCH("delta_head_prepare");
    return GK_OK;
}

}  // namespace

// proj: the mixer's first column in every row.  conv_w [taps, C], ring [slots, taps, C] 32-bit.  rounded = 0: q, k, v are 32-bit
// and g the decay factors; rounded = 1: q, k, v are bfloat16, q_unit, k_unit [T, G] their factors and g the logarithms.
GK_EXPORT int gk_delta_head_prepare(const void* proj, int dtype, long long ld, const float* conv_w, const float* ring,
                                    const float* a_log, const float* dt_bias, const int* tok_pos, const int* tok_seq,
                                    const int* cu_q, const int* slots, void* q, void* k, void* v, float* q_unit, float* k_unit,
                                    float* g, float* beta, int rounded, int n_tokens, int n_heads, int n_kv, int d, int dv, int taps,
                                    void* stream) {
    GK_REQUIRE(GK_VALID_DTYPE(dtype), "delta_head_prepare: bad dtype");
    GK_REQUIRE(sizes_ok(n_heads, n_kv, d, dv, taps), "delta_head_prepare: bad sizes (1 to %d taps)", MAX_TAPS);
    GK_REQUIRE(taps == 1 || ring != nullptr, "delta_head_prepare: a convolution of several taps needs its state");
    GK_REQUIRE(d <= 512 && dv <= 512, "delta_head_prepare: heads of %d / %d are more than a warp holds (512)", d, dv);
    GK_REQUIRE(!rounded || (dtype == GK_BF16 && q_unit != nullptr && k_unit != nullptr),
               "delta_head_prepare: rounded vectors come from a bfloat16 projection and with their factors");
    if (n_tokens == 0) return GK_OK;
    const HeadSizes sz{n_heads, n_kv, d, dv, taps};
    cudaStream_t s = (cudaStream_t)stream;
    const uintptr_t all = (uintptr_t)proj | (uintptr_t)conv_w | (uintptr_t)ring | (uintptr_t)q | (uintptr_t)k | (uintptr_t)v;
    const bool vec = d % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && (all & 15) == 0;
#define GK_PREP_AS(TO, VEC, TAPS)                                                                                              \
    return prepare_as<T, TO, VEC, TAPS>(proj, ld, conv_w, ring, a_log, dt_bias, tok_pos, tok_seq, cu_q, slots,                 \
                                        PrepareOut<TO>{(TO*)q, (TO*)k, (TO*)v, q_unit, k_unit, g, beta}, n_tokens, sz, s)
#define GK_PREP(TO)                                \
    do {                                           \
        if (vec && taps == 4) GK_PREP_AS(TO, 4, 4); \
        if (vec) GK_PREP_AS(TO, 4, 0);             \
        GK_PREP_AS(TO, 1, 0);                      \
    } while (0)
    if (rounded) {
        using T = __nv_bfloat16;
        GK_PREP(__nv_bfloat16);
    }
    GK_DISPATCH_DTYPE(dtype, T, { GK_PREP(float); })
#undef GK_PREP
#undef GK_PREP_AS
    return GK_OK;
}

// kv_len[i]: the sequence's tokens including this step's
GK_EXPORT int gk_conv_ring(const void* proj, int dtype, long long ld, float* ring, const int* cu_q, const int* kv_len, const int* slots,
                           int n_seqs, int channels, int taps, void* stream) {
    GK_REQUIRE(GK_VALID_DTYPE(dtype), "conv_ring: bad dtype %d", dtype);
    GK_REQUIRE(taps >= 1 && channels > 0 && n_seqs <= 65535, "conv_ring: bad sizes");
    if (n_seqs == 0 || taps == 1) return GK_OK;
    cudaStream_t s = (cudaStream_t)stream;
    GK_DISPATCH_DTYPE(dtype, T, {
        gk_launch(conv_ring_kernel<T>, dim3((channels + 255) / 256, n_seqs), dim3(256), 0, s, (const T*)proj, ld, ring, cu_q, kv_len, slots,
                  channels, taps);
    })
    GK_CHECK_LAUNCH("conv_ring");
    return GK_OK;
}

// Threads, column groups and rows a thread for heads of these sizes; 0 where no block holds the state in registers.
static int single_shape(int d, int dv) {
    if (d <= 0 || dv <= 0 || dv % 4 != 0) return 0;
    if (dv <= 32) return d <= 128 ? 1 : d <= 256 ? 2 : 0;
    if (dv <= 64) return d <= 128 ? 3 : d <= 256 ? 4 : 0;
    if (dv <= 128) return d <= 64 ? 5 : d <= 128 ? 6 : d <= 256 ? 7 : 0;
    if (dv <= 256) return d <= 128 ? 8 : 0;
    return 0;
}

GK_EXPORT int gk_delta_head_single_fits(int d, int dv) { return single_shape(d, dv) != 0; }

// proj: the mixer's first column in every row (row t is the token of sequence tok_seq[t]); norm_w [dv]; a head's result, times
// out_scale, is at columns h dv .. of the token's row of `out`, rows ld_out apart.
GK_EXPORT int gk_delta_head_single(const void* proj, int dtype, long long ld, const float* conv_w, float* ring, const float* a_log,
                                   const float* dt_bias, const float* norm_w, float* state, const int* tok_pos, const int* tok_seq,
                                   const int* slots, void* out, long long ld_out, float out_scale, float eps, int n_tokens, int n_heads,
                                   int n_kv, int d, int dv, int taps, void* stream) {
    GK_REQUIRE(GK_VALID_DTYPE(dtype), "delta_head_single: bad dtype");
    GK_REQUIRE(sizes_ok(n_heads, n_kv, d, dv, taps) && n_tokens <= 65535 && eps > 0.f, "delta_head_single: bad sizes");
    GK_REQUIRE(taps == 1 || ring != nullptr, "delta_head_single: a convolution of several taps needs its state");
    const int shape = single_shape(d, dv);
    GK_REQUIRE(shape != 0, "delta_head_single: heads of %d / %d do not fit a block", d, dv);
    GK_REQUIRE(((uintptr_t)state & 15) == 0, "delta_head_single: the state must start on 16 bytes");
    if (n_tokens == 0) return GK_OK;
    const HeadSizes sz{n_heads, n_kv, d, dv, taps};
    cudaStream_t s = (cudaStream_t)stream;
    const size_t vectors = (size_t)(2 * ((d + 3) & ~3) + 2 * ((dv + 3) & ~3)) * sizeof(float);
#define GK_SINGLE_AS(NT, CG, R, TAPS)                                                                                                       \
    gk_launch(delta_head_single_kernel<T, NT, CG, R, TAPS>, dim3(n_heads, n_tokens), dim3(NT), vectors + (size_t)NT * 8 * sizeof(float), s, \
              (const T*)proj, ld, conv_w, ring, a_log, dt_bias, norm_w, state, tok_pos, tok_seq, slots, (T*)out, ld_out, out_scale, eps, sz)
#define GK_SINGLE(NT, CG, R)                     \
    do {                                         \
        if (taps == 4) GK_SINGLE_AS(NT, CG, R, 4); \
        else GK_SINGLE_AS(NT, CG, R, 0);         \
    } while (0)
    GK_DISPATCH_DTYPE(dtype, T, {
        switch (shape) {
            case 1: GK_SINGLE(256, 8, 4); break;
            case 2: GK_SINGLE(256, 8, 8); break;
            case 3: GK_SINGLE(256, 16, 8); break;
            case 4: GK_SINGLE(256, 16, 16); break;
            case 5: GK_SINGLE(256, 32, 8); break;
            case 6: GK_SINGLE(256, 32, 16); break;
            case 7: GK_SINGLE(512, 32, 16); break;
            default: GK_SINGLE(512, 64, 16); break;
        }
    })
#undef GK_SINGLE
#undef GK_SINGLE_AS
    GK_CHECK_LAUNCH("delta_head_single");
    return GK_OK;
}

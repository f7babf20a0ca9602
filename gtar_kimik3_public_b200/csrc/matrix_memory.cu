// The recurrence of a matrix memory with an exponential input gate and a forget gate (the mLSTM of xLSTM), token by token:
//
//   i = cap tanh((z_i + b_i) / cap) ;  f = logsigmoid(cap tanh((z_f + b_f) / cap))                     per token and head
//   m' = max(f + m, i) ;  C <- e^(f + m - m') C + e^(i - m') k v^T ;  n <- e^(f + m - m') n + e^(i - m') k
//   num = C^T q ;  den = max(|n . q|, e^(-m')) + 1e-6                                                 (o = num / den)
//
// The kernels read the packed projection as it is (columns of q, k, v, z_i, z_f; k times d^(-1/2) as it is loaded) and write num
// [T, H, dv] and den [T, H] in 32-bit; the norm behind them divides.  n is treated as one more column of C whose value is 1.
// The state in memory: C with one more row [slots, H, d + 1, dv] and n with one more entry [slots, H, d + 1]; the extra
// row and entry hold m, a copy for every column, so blocks that own different columns never touch one another's numbers.

#include "matrix_memory.cuh"

namespace {

using namespace memory;

constexpr int LANES = 8;      // lanes that share a column of the state
constexpr int MAX_COLS = 32;  // columns a block at most (256 threads)

// A column's d entries are spread over eight adjacent lanes, R consecutive rows a lane; TB tokens are staged at a time.
template <typename T, int R, int TB>
__global__ void __launch_bounds__(LANES * MAX_COLS) memory_scan_kernel(
    const T* __restrict__ proj, long long ld, Columns at, const float* __restrict__ gate_bias, float cap, float k_scale,
    float* __restrict__ state, float* __restrict__ n_state, float* __restrict__ out, float* __restrict__ den,
    const int* __restrict__ cu_q, const int* __restrict__ slots, int n_heads, int d, int dv) {
    constexpr int PIECE = R == 4 ? 4 : R + 4, VEC = LANES * PIECE;  // a lane's piece starts a bank group apart from its neighbours'
    __shared__ __align__(16) float sq[TB][VEC], sk[TB][VEC];
    __shared__ float sv[TB][MAX_COLS];
    __shared__ float s_old[TB], s_new[TB], s_top[TB];
    pdl_launch_dependents();
    const int n_threads = blockDim.x, n_cols = n_threads / LANES;
    const int seq = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * n_cols;
    const int sub = threadIdx.x % LANES, col = col0 + threadIdx.x / LANES;
    const bool live = col <= dv;   // column dv is n
    const bool is_n = col == dv;
    for (int i = threadIdx.x; i < TB * VEC; i += n_threads) {  // the pieces beyond d stay zero
        (&sq[0][0])[i] = 0.f;
        (&sk[0][0])[i] = 0.f;
    }
    const float bias_i = gate_bias[head], bias_f = gate_bias[n_heads + head];
    pdl_wait();
    const int t0 = cu_q[seq], n = cu_q[seq + 1] - t0;
    const size_t slot_head = (size_t)slots[seq] * n_heads + head;
    float* column = is_n ? n_state + slot_head * (d + 1) : state + slot_head * (d + 1) * dv + col;
    const size_t stride = is_n ? 1 : dv;
    float S[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int row = sub * R + r;
        S[r] = (live && row < d) ? column[(size_t)row * stride] : 0.f;
    }
    float top = live ? column[(size_t)d * stride] : 0.f;  // the same number in every column
    for (int first = 0; first < n; first += TB) {
        const int count = min(TB, n - first);
        __syncthreads();  // the tokens of before are done with
        for (int i = threadIdx.x; i < count * d; i += n_threads) {
            const int tt = i / d, c = i - tt * d;
            const int to = (c / R) * PIECE + c % R;
            const T* row = proj + (size_t)(t0 + first + tt) * ld;
            sq[tt][to] = to_float(row[at.q + head * d + c]);
            sk[tt][to] = to_float(row[at.k + head * d + c]) * k_scale;
        }
        for (int i = threadIdx.x; i < count * n_cols; i += n_threads) {
            const int tt = i / n_cols, cc = i - tt * n_cols;
            const int vc = col0 + cc;
            sv[tt][cc] = vc < dv ? to_float(proj[(size_t)(t0 + first + tt) * ld + at.v + head * dv + vc]) : vc == dv ? 1.f : 0.f;
        }
        for (int tt = threadIdx.x; tt < count; tt += n_threads) {
            const T* row = proj + (size_t)(t0 + first + tt) * ld;
            s_new[tt] = log_input_gate(to_float(row[at.i + head]) + bias_i, cap);
            s_old[tt] = log_forget_gate(to_float(row[at.f + head]) + bias_f, cap);
        }
        __syncthreads();
        if (threadIdx.x == 0) {  // the running maximum, one token after another
            float m = top;
            for (int tt = 0; tt < count; ++tt) {
                const float f = s_old[tt], i = s_new[tt], m_new = fmaxf(f + m, i);
                s_old[tt] = f + m - m_new;
                s_new[tt] = i - m_new;
                s_top[tt] = m = m_new;
            }
        }
        __syncthreads();
        for (int tt = threadIdx.x; tt < 2 * count; tt += n_threads) {
            if (tt < count) s_old[tt] = expf(s_old[tt]);
            else s_new[tt - count] = expf(s_new[tt - count]);
        }
        __syncthreads();
        top = s_top[count - 1];
        const float4* pq = reinterpret_cast<const float4*>(&sq[0][sub * PIECE]);
        const float4* pk = reinterpret_cast<const float4*>(&sk[0][sub * PIECE]);
        for (int tt = 0; tt < count; ++tt, pq += VEC / 4, pk += VEC / 4) {
            const float keep = s_old[tt], vv = s_new[tt] * sv[tt][threadIdx.x / LANES];
            float b4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int r4 = 0; r4 < R / 4; ++r4) {
                const float4 k4 = pk[r4], q4 = pq[r4];
                const float ks[4] = {k4.x, k4.y, k4.z, k4.w}, qs[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int r = 4 * r4 + e;
                    S[r] = fmaf(ks[e], vv, keep * S[r]);
                    b4[e] = fmaf(S[r], qs[e], b4[e]);
                }
            }
            float b = (b4[0] + b4[1]) + (b4[2] + b4[3]);
#pragma unroll
            for (int o = 1; o < LANES; o <<= 1) b += __shfl_xor_sync(0xffffffffu, b, o);
            if (live && sub == 0) {
                const size_t row = (size_t)(t0 + first + tt) * n_heads + head;
                if (is_n) den[row] = fmaxf(fabsf(b), expf(-s_top[tt])) + DEN_ADD;
                else out[row * dv + col] = b;
            }
        }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int row = sub * R + r;
        if (live && row < d) column[(size_t)row * stride] = S[r];
    }
    if (live && sub == 0) column[(size_t)d * stride] = top;
}

}  // namespace

GK_EXPORT int gk_memory_scan(const void* proj, int dtype, long long ld, int q_at, int k_at, int v_at, int i_at, int f_at,
                             const float* gate_bias, float cap, float* state, float* n_state, float* out, float* den, const int* cu_q,
                             const int* slots, int n_seqs, int n_heads, int d, int dv, void* stream) {
    GK_REQUIRE(GK_VALID_DTYPE(dtype), "memory_scan: bad dtype %d", dtype);
    GK_REQUIRE(n_heads > 0 && n_heads <= 65535 && n_seqs >= 0 && n_seqs <= 65535, "memory_scan: bad counts");
    GK_REQUIRE(d > 0 && d <= 512 && dv > 0, "memory_scan: key size %d must be at most 512, value size %d positive", d, dv);
    GK_REQUIRE(cap > 0.f, "memory_scan: the gates' cap must be positive");
    if (n_seqs == 0) return GK_OK;
    const int sms = memory::sm_count();
    // fewer columns a block while the blocks do not fill the device twice: a column's sums do not depend on the block's shape
    int cols = MAX_COLS;
    while (cols > 4 && (long long)n_seqs * n_heads * ((dv + cols) / cols) < 2LL * sms) cols /= 2;
    const dim3 grid((dv + cols) / cols, n_heads, n_seqs), block(cols * LANES);  // dv + 1 columns, rounded up
    const memory::Columns at = {q_at, k_at, v_at, i_at, f_at};
    const float k_scale = 1.f / sqrtf((float)d);
    cudaStream_t s = (cudaStream_t)stream;
#define GK_SCAN(R, TB)                                                                                                               \
    gk_launch(memory_scan_kernel<T, R, TB>, grid, block, 0, s, (const T*)proj, ld, at, gate_bias, cap, k_scale, state, n_state, out, den, \
              cu_q, slots, n_heads, d, dv)
    GK_DISPATCH_DTYPE(dtype, T, {
        if (d <= 32) GK_SCAN(4, 16);
        else if (d <= 64) GK_SCAN(8, 16);
        else if (d <= 128) GK_SCAN(16, 16);
        else if (d <= 256) GK_SCAN(32, 8);
        else GK_SCAN(64, 4);
    })
#undef GK_SCAN
    GK_CHECK_LAUNCH("memory_scan");
    return GK_OK;
}

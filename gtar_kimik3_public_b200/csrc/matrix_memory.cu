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
//
// memory_single is the step of one token a sequence with the norm of the head, its weight and the sigmoid gate in the same
// kernel: a cluster of blocks per (sequence, head), 64 value columns a block, one exchange of the blocks' sums of squares.

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

constexpr int ONE_THREADS = 256, ONE_COLS = 64, ONE_LANES = ONE_COLS / 4, ONE_GROUPS = ONE_THREADS / ONE_LANES;

// Sixteen threads side by side own four columns each, sixteen groups of them every sixteenth row (R rows a group): a thread
// has all its rows' loads in flight at once.  n is updated by every block for itself, written by the cluster's first block once
// all of them have read it.
template <typename T, int R>
__global__ void __launch_bounds__(ONE_THREADS) memory_single_kernel(
    const T* __restrict__ proj, long long ld, Columns at, int g_at, const float* __restrict__ gate_bias, float cap, float k_scale,
    float* __restrict__ state, float* __restrict__ n_state, const float* __restrict__ norm_w, float eps, T* __restrict__ y,
    const int* __restrict__ cu_q, const int* __restrict__ slots, int n_heads, int d, int dv) {
    constexpr int D = R * ONE_GROUPS, PER = (D + ONE_THREADS - 1) / ONE_THREADS;
    __shared__ float sq[D], sk[D];
    __shared__ __align__(16) float part[ONE_GROUPS][ONE_COLS];
    __shared__ float scratch[33];
    __shared__ float squares[8];  // of every block of the cluster
    pdl_launch_dependents();
    asm volatile("barrier.cluster.arrive.relaxed.aligned;" ::: "memory");  // the other blocks run: their memory may be written
    const int tile = blockIdx.x, tiles = gridDim.x, head = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x;
    const int lane4 = tid % ONE_LANES, grp = tid / ONE_LANES;
    const int col = tile * ONE_COLS + lane4 * 4;
    const bool live = col < dv;
    const float bias_i = gate_bias[head], bias_f = gate_bias[n_heads + head];
    pdl_wait();
    const int t = cu_q[seq];
    const size_t slot_head = (size_t)slots[seq] * n_heads + head;
    float* own = state + slot_head * (size_t)(d + 1) * dv + col;
    float* own_n = n_state + slot_head * (d + 1);
    float4 S[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int row = grp + r * ONE_GROUPS;
        S[r] = live && row < d ? *reinterpret_cast<const float4*>(own + (size_t)row * dv) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const T* row = proj + (size_t)t * ld;
    float n_new[PER];
    const float m = own_n[d];
    const float i = log_input_gate(to_float(row[at.i + head]) + bias_i, cap);
    const float f = log_forget_gate(to_float(row[at.f + head]) + bias_f, cap);
    const float m_new = fmaxf(f + m, i), keep = expf(f + m - m_new), in = expf(i - m_new);
    float dot = 0.f;
#pragma unroll
    for (int p = 0; p < PER; ++p) {
        const int e = tid + p * ONE_THREADS;
        n_new[p] = 0.f;
        if (e < D) {
            const float q = e < d ? to_float(row[at.q + head * d + e]) : 0.f;
            const float k = e < d ? to_float(row[at.k + head * d + e]) * k_scale : 0.f;
            sq[e] = q;
            sk[e] = k * in;
            if (e < d) n_new[p] = fmaf(in, k, keep * own_n[e]);
            dot = fmaf(q, n_new[p], dot);
        }
    }
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live) {
        const T* vr = row + at.v + head * dv + col;
        v = make_float4(to_float(vr[0]), to_float(vr[1]), to_float(vr[2]), to_float(vr[3]));
    }
    dot = block_sum(dot, scratch);  // its barriers also publish sq and sk
    const float inv = 1.f / (fmaxf(fabsf(dot), expf(-m_new)) + DEN_ADD);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int at_row = grp + r * ONE_GROUPS;
        const float k = sk[at_row], q = sq[at_row];
        S[r].x = fmaf(k, v.x, keep * S[r].x), S[r].y = fmaf(k, v.y, keep * S[r].y);
        S[r].z = fmaf(k, v.z, keep * S[r].z), S[r].w = fmaf(k, v.w, keep * S[r].w);
        o.x = fmaf(q, S[r].x, o.x), o.y = fmaf(q, S[r].y, o.y), o.z = fmaf(q, S[r].z, o.z), o.w = fmaf(q, S[r].w, o.w);
        if (live && at_row < d) *reinterpret_cast<float4*>(own + (size_t)at_row * dv) = S[r];
    }
    *reinterpret_cast<float4*>(&part[grp][lane4 * 4]) = o;
    __syncthreads();
    float num = 0.f;
    if (tid < ONE_COLS) {
#pragma unroll
        for (int gi = 0; gi < ONE_GROUPS; ++gi) num += part[gi][tid];
        num *= inv;
    }
    const float ss = block_sum(num * num, scratch);
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (tid < tiles) {
        uint32_t remote;
        asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"((uint32_t)__cvta_generic_to_shared(&squares[tile])), "r"(tid));
        asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(ss) : "memory");
    }
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (tile == 0) {
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int e = tid + p * ONE_THREADS;
            if (e < d) own_n[e] = n_new[p];
        }
        if (tid == 0) own_n[d] = m_new;
    }
    const int mine = tile * ONE_COLS + tid;
    if (tid < ONE_COLS && mine < dv) {
        float total = 0.f;
        for (int w = 0; w < tiles; ++w) total += squares[w];
        const float r = 1.f / sqrtf(total / (float)dv + eps);
        const float z = to_float(row[g_at + head * dv + mine]);
        y[(size_t)t * n_heads * dv + head * dv + mine] = from_float<T>(num * r * norm_w[head * dv + mine] / (1.f + expf(-z)));
        state[slot_head * (size_t)(d + 1) * dv + (size_t)d * dv + mine] = m_new;
    }
}

}  // namespace

// One token a sequence: the recurrence, the heads' norm and the gate.  y [n_tokens, H dv] in the run's type.
GK_EXPORT int gk_memory_single(const void* proj, int dtype, long long ld, int q_at, int k_at, int v_at, int g_at, int i_at, int f_at,
                               const float* gate_bias, float cap, float* state, float* n_state, const float* norm_w, float eps, void* y,
                               const int* cu_q, const int* slots, int n_seqs, int n_heads, int d, int dv, void* stream) {
    GK_REQUIRE(GK_VALID_DTYPE(dtype), "memory_single: bad dtype %d", dtype);
    GK_REQUIRE(n_heads > 0 && n_heads <= 65535 && n_seqs >= 0 && n_seqs <= 65535, "memory_single: bad counts");
    GK_REQUIRE(d > 0 && d <= 512 && dv > 0 && dv % 4 == 0 && dv <= 8 * ONE_COLS, "memory_single: heads of %d / %d do not fit", d, dv);
    GK_REQUIRE(cap > 0.f && eps > 0.f, "memory_single: cap and eps must be positive");
    if (n_seqs == 0) return GK_OK;
    const int tiles = (dv + ONE_COLS - 1) / ONE_COLS;
    const memory::Columns at = {q_at, k_at, v_at, i_at, f_at};
    const float k_scale = 1.f / sqrtf((float)d);
    cudaStream_t s = (cudaStream_t)stream;
#define GK_ONE(R)                                                                                                                    \
    gk_launch_cluster(memory_single_kernel<T, R>, dim3(tiles, n_heads, n_seqs), dim3(ONE_THREADS), 0, s, dim3(tiles, 1, 1), (const T*)proj, \
                      ld, at, g_at, gate_bias, cap, k_scale, state, n_state, norm_w, eps, (T*)y, cu_q, slots, n_heads, d, dv)
    GK_DISPATCH_DTYPE(dtype, T, {
        if (d <= 64) GK_ONE(4);
        else if (d <= 128) GK_ONE(8);
        else if (d <= 256) GK_ONE(16);
        else GK_ONE(32);
    })
#undef GK_ONE
    GK_CHECK_LAUNCH("memory_single");
    return GK_OK;
}

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

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
// memory_single is the bfloat16 step of one token a sequence with the norm of the head, its weight and the sigmoid gate in the same
// kernel: a cluster of blocks per (sequence, head), 64 value columns a block, one exchange of the blocks' sums of squares.

#include "matrix_memory.cuh"

namespace {

using namespace memory;

constexpr int LANES = 8;      // lanes that share a column of the state
constexpr int MAX_COLS = 32;  // columns a block at most (256 threads)

// The gates of a sequence's tokens, a warp per (sequence, head): gates [T, H] = (e^(f + m - m'), e^(i - m'), m', 0).  The running
// maximum goes from token to token in order, so it does not depend on how a prompt is cut.
template <typename T>
__global__ void __launch_bounds__(32) memory_gates_kernel(const T* __restrict__ proj, long long ld, Columns at,
                                                          const float* __restrict__ gate_bias, float cap, const float* __restrict__ n_state,
                                                          float4* __restrict__ gates, const int* __restrict__ cu_q,
                                                          const int* __restrict__ slots, int n_heads, int d) {
    pdl_launch_dependents();
    const int head = blockIdx.x, seq = blockIdx.y, lane = threadIdx.x;
    const float bias_i = gate_bias[head], bias_f = gate_bias[n_heads + head];
    pdl_wait();
    const int t0 = cu_q[seq], n = cu_q[seq + 1] - t0;
    if (n <= 0) return;
    float m = n_state[((size_t)slots[seq] * n_heads + head) * (d + 1) + d];
    float z_i = 0.f, z_f = 0.f;
    auto fetch = [&](int first) {
        if (first + lane < n) {
            const T* row = proj + (size_t)(t0 + first + lane) * ld;
            z_i = to_float(row[at.i + head]);
            z_f = to_float(row[at.f + head]);
        }
    };
    fetch(0);
    for (int first = 0; first < n; first += 32) {
        const float i = log_input_gate(z_i + bias_i, cap), f = log_forget_gate(z_f + bias_f, cap);
        if (first + 32 < n) fetch(first + 32);
        const int count = min(32, n - first);
        float before = 0.f, after = 0.f;
#pragma unroll 8
        for (int tt = 0; tt < count; ++tt) {
            const float fi = __shfl_sync(0xffffffffu, f, tt), ii = __shfl_sync(0xffffffffu, i, tt);
            const float m_new = fmaxf(fi + m, ii);
            if (lane == tt) {
                before = m;
                after = m_new;
            }
            m = m_new;
        }
        if (lane < count) gates[(size_t)(t0 + first + lane) * n_heads + head] = make_float4(expf(f + before - after), expf(i - after), after, 0.f);
    }
}

template <int BYTES>
__device__ __forceinline__ void copy_async(void* smem, const void* gmem) {
    if constexpr (BYTES == 16)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem));
    else
        asm volatile("cp.async.ca.shared.global [%0], [%1], %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(smem)), "l"(gmem), "n"(BYTES));
}

// 16 bytes of a row in shared memory as 32-bit numbers
__device__ __forceinline__ void row_piece(const float* p, float (&v)[4]) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
}
__device__ __forceinline__ void row_piece(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int c = 0; c < 4; ++c) {
        const float2 x = __bfloat1622float2(h[c]);
        v[2 * c] = x.x, v[2 * c + 1] = x.y;
    }
}

// A column's d entries are spread over eight adjacent lanes, R consecutive rows a lane.  The step's tokens come through a
// two-stage cp.async ring, TB at a time, in the projection's type (VEC: its rows and their parts are whole 16-byte pieces).
template <typename T, int R, int TB, bool VEC>
__global__ void __launch_bounds__(LANES * MAX_COLS) memory_scan_kernel(
    const T* __restrict__ proj, long long ld, Columns at, const float4* __restrict__ gates, float k_scale, float* __restrict__ state,
    float* __restrict__ n_state, float* __restrict__ out, float* __restrict__ den, const int* __restrict__ cu_q,
    const int* __restrict__ slots, int n_heads, int d, int dv) {
    constexpr int PER16 = 16 / sizeof(T);
    constexpr int PIECE = R + PER16, ROW = LANES * PIECE;  // a lane's piece starts a bank group apart from its neighbours'
    static_assert(R % PER16 == 0, "a lane's rows are whole pieces");
    __shared__ __align__(16) T sq[2][TB][ROW], sk[2][TB][ROW];
    __shared__ __align__(16) T sv[2][TB][MAX_COLS];
    __shared__ float4 sg[2][TB];
    pdl_launch_dependents();
    const int n_threads = blockDim.x, n_cols = n_threads / LANES;
    const int seq = blockIdx.z, head = blockIdx.y, col0 = blockIdx.x * n_cols;
    const int sub = threadIdx.x % LANES, my_col = threadIdx.x / LANES, col = col0 + my_col;
    const bool live = col <= dv;   // column dv is n
    const bool is_n = col == dv;
    for (int i = threadIdx.x; i < 2 * TB * ROW; i += n_threads) {  // the pieces beyond d stay zero
        (&sq[0][0][0])[i] = from_float<T>(0.f);
        (&sk[0][0][0])[i] = from_float<T>(0.f);
    }
    __syncthreads();
    pdl_wait();
    const int t0 = cu_q[seq], n = cu_q[seq + 1] - t0;
    if (n <= 0) return;
    const size_t slot_head = (size_t)slots[seq] * n_heads + head;
    float* column = is_n ? n_state + slot_head * (d + 1) : state + slot_head * (d + 1) * dv + col;
    const size_t stride = is_n ? 1 : dv;
    float S[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        const int row = sub * R + r;
        S[r] = (live && row < d) ? column[(size_t)row * stride] : 0.f;
    }
    auto stage = [&](int buf, int first) {
        const int count = min(TB, n - first);
        const T* row0 = proj + (size_t)(t0 + first) * ld + head * d;
        const T* v0 = proj + (size_t)(t0 + first) * ld + at.v + head * dv + col0;
        if constexpr (VEC) {
            const int pieces = d / PER16;
            for (int i = threadIdx.x; i < count * pieces; i += n_threads) {
                const int tt = i / pieces, c = (i - tt * pieces) * PER16, to = (c / R) * PIECE + c % R;
                copy_async<16>(&sq[buf][tt][to], row0 + (size_t)tt * ld + at.q + c);
                copy_async<16>(&sk[buf][tt][to], row0 + (size_t)tt * ld + at.k + c);
            }
            const int quads = n_cols / 4;
            for (int i = threadIdx.x; i < count * quads; i += n_threads) {
                const int tt = i / quads, c = (i - tt * quads) * 4;
                if (col0 + c < dv) copy_async<4 * sizeof(T)>(&sv[buf][tt][c], v0 + (size_t)tt * ld + c);
            }
        } else {
            for (int i = threadIdx.x; i < count * d; i += n_threads) {
                const int tt = i / d, c = i - tt * d, to = (c / R) * PIECE + c % R;
                sq[buf][tt][to] = row0[(size_t)tt * ld + at.q + c];
                sk[buf][tt][to] = row0[(size_t)tt * ld + at.k + c];
            }
            for (int i = threadIdx.x; i < count * n_cols; i += n_threads) {
                const int tt = i / n_cols, c = i - tt * n_cols;
                if (col0 + c < dv) sv[buf][tt][c] = v0[(size_t)tt * ld + c];
            }
        }
        for (int tt = threadIdx.x; tt < count; tt += n_threads) copy_async<16>(&sg[buf][tt], gates + (size_t)(t0 + first + tt) * n_heads + head);
        asm volatile("cp.async.commit_group;\n" ::);
    };
    stage(0, 0);
    float top = 0.f;
    int buf = 0;
    for (int first = 0; first < n; first += TB, buf ^= 1) {
        if (first + TB < n) {
            stage(buf ^ 1, first + TB);
            asm volatile("cp.async.wait_group 1;\n" ::);
        } else {
            asm volatile("cp.async.wait_group 0;\n" ::);
        }
        __syncthreads();
        const int count = min(TB, n - first);
#pragma unroll 2
        for (int tt = 0; tt < count; ++tt) {
            const float4 g = sg[buf][tt];
            const float v = is_n ? 1.f : live ? to_float(sv[buf][tt][my_col]) : 0.f;
            const float vv = g.y * k_scale * v;
            float b4[4] = {0.f, 0.f, 0.f, 0.f};  // four partial sums: chains of R / 4 dependent operations
#pragma unroll
            for (int r0 = 0; r0 < R; r0 += PER16) {
                float ks[PER16], qs[PER16];
                row_piece(&sk[buf][tt][sub * PIECE + r0], ks);
                row_piece(&sq[buf][tt][sub * PIECE + r0], qs);
#pragma unroll
                for (int e = 0; e < PER16; ++e) {
                    S[r0 + e] = fmaf(ks[e], vv, g.x * S[r0 + e]);
                    b4[e & 3] = fmaf(S[r0 + e], qs[e], b4[e & 3]);
                }
            }
            float b = (b4[0] + b4[1]) + (b4[2] + b4[3]);
#pragma unroll
            for (int o = 1; o < LANES; o <<= 1) b += __shfl_xor_sync(0xffffffffu, b, o);
            if (live && sub == 0) {
                const size_t row = (size_t)(t0 + first + tt) * n_heads + head;
                if (is_n) den[row] = fmaxf(fabsf(b), expf(-g.z)) + DEN_ADD;
                else out[row * dv + col] = b;
            }
            top = g.z;
        }
        __syncthreads();  // the stage is free for the load after next
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
template <int R>
__global__ void __launch_bounds__(ONE_THREADS) memory_single_kernel(
    const __nv_bfloat16* __restrict__ proj, long long ld, Columns at, int g_at, const float* __restrict__ gate_bias, float cap, float k_scale,
    float* __restrict__ state, float* __restrict__ n_state, const float* __restrict__ norm_w, float eps, __nv_bfloat16* __restrict__ y,
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
    const __nv_bfloat16* row = proj + (size_t)t * ld;
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
        const __nv_bfloat16* vr = row + at.v + head * dv + col;
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
        y[(size_t)t * n_heads * dv + head * dv + mine] = __float2bfloat16_rn(num * r * norm_w[head * dv + mine] / (1.f + expf(-z)));
        state[slot_head * (size_t)(d + 1) * dv + (size_t)d * dv + mine] = m_new;
    }
}

}  // namespace

// One token a sequence: the recurrence, the heads' norm and the gate, bfloat16 rows; y [n_tokens, H dv].
GK_EXPORT int gk_memory_single(const void* proj, long long ld, int q_at, int k_at, int v_at, int g_at, int i_at, int f_at,
                               const float* gate_bias, float cap, float* state, float* n_state, const float* norm_w, float eps, void* y,
                               const int* cu_q, const int* slots, int n_seqs, int n_heads, int d, int dv, void* stream) {
    GK_REQUIRE(n_heads > 0 && n_heads <= 65535 && n_seqs >= 0 && n_seqs <= 65535, "memory_single: bad counts");
    GK_REQUIRE(d > 0 && d <= 512 && dv > 0 && dv % 4 == 0 && dv <= 8 * ONE_COLS, "memory_single: heads of %d / %d do not fit", d, dv);
    GK_REQUIRE(cap > 0.f && eps > 0.f, "memory_single: cap and eps must be positive");
    if (n_seqs == 0) return GK_OK;
    const int tiles = (dv + ONE_COLS - 1) / ONE_COLS;
    const memory::Columns at = {q_at, k_at, v_at, i_at, f_at};
    const float k_scale = 1.f / sqrtf((float)d);
    cudaStream_t s = (cudaStream_t)stream;
#define GK_ONE(R)                                                                                                                    \
    gk_launch_cluster(memory_single_kernel<R>, dim3(tiles, n_heads, n_seqs), dim3(ONE_THREADS), 0, s, dim3(tiles, 1, 1), (const __nv_bfloat16*)proj, \
                      ld, at, g_at, gate_bias, cap, k_scale, state, n_state, norm_w, eps, (__nv_bfloat16*)y, cu_q, slots, n_heads, d, dv)
    if (d <= 64) GK_ONE(4);
    else if (d <= 128) GK_ONE(8);
    else if (d <= 256) GK_ONE(16);
    else GK_ONE(32);
#undef GK_ONE
    GK_CHECK_LAUNCH("memory_single");
    return GK_OK;
}

// `gates` holds n_tokens * H * 4 floats.
GK_EXPORT int gk_memory_scan(const void* proj, int dtype, long long ld, int q_at, int k_at, int v_at, int i_at, int f_at,
                             const float* gate_bias, float cap, float* state, float* n_state, float* gates, float* out, float* den,
                             const int* cu_q, const int* slots, int n_seqs, int n_heads, int d, int dv, void* stream) {
    GK_REQUIRE(GK_VALID_DTYPE(dtype), "memory_scan: bad dtype %d", dtype);
    GK_REQUIRE(n_heads > 0 && n_heads <= 65535 && n_seqs >= 0 && n_seqs <= 65535, "memory_scan: bad counts");
    GK_REQUIRE(d > 0 && d <= 512 && dv > 0, "memory_scan: key size %d must be at most 512, value size %d positive", d, dv);
    GK_REQUIRE(cap > 0.f && reinterpret_cast<uintptr_t>(gates) % 16 == 0, "memory_scan: the gates' cap must be positive, their array aligned");
    if (n_seqs == 0) return GK_OK;
    const int sms = memory::sm_count();
    // fewer columns a block while the blocks do not fill the device twice: a column's sums do not depend on the block's shape
    int cols = MAX_COLS;
    while (cols > 4 && (long long)n_seqs * n_heads * ((dv + cols) / cols) < 2LL * sms) cols /= 2;
    const dim3 grid((dv + cols) / cols, n_heads, n_seqs), block(cols * LANES);  // dv + 1 columns, rounded up
    const memory::Columns at = {q_at, k_at, v_at, i_at, f_at};
    const float k_scale = 1.f / sqrtf((float)d);
    const int per16 = dtype == GK_F32 ? 4 : 8;
    const bool vec = d % per16 == 0 && dv % 4 == 0 && ld % per16 == 0 && q_at % per16 == 0 && k_at % per16 == 0 && v_at % 4 == 0 &&
                     reinterpret_cast<uintptr_t>(proj) % 16 == 0;
    cudaStream_t s = (cudaStream_t)stream;
#define GK_SCAN(R, TB)                                                                                                               \
    do {                                                                                                                             \
        if (vec)                                                                                                                     \
            gk_launch(memory_scan_kernel<T, R, TB, true>, grid, block, 0, s, (const T*)proj, ld, at, (const float4*)gates, k_scale,  \
                      state, n_state, out, den, cu_q, slots, n_heads, d, dv);                                                        \
        else                                                                                                                         \
            gk_launch(memory_scan_kernel<T, R, TB, false>, grid, block, 0, s, (const T*)proj, ld, at, (const float4*)gates, k_scale, \
                      state, n_state, out, den, cu_q, slots, n_heads, d, dv);                                                        \
    } while (0)
    GK_DISPATCH_DTYPE(dtype, T, {
        gk_launch(memory_gates_kernel<T>, dim3(n_heads, n_seqs), dim3(32), 0, s, (const T*)proj, ld, at, gate_bias, cap, (const float*)n_state,
                  (float4*)gates, cu_q, slots, n_heads, d);
        GK_CHECK_LAUNCH("memory_gates");
        if (d <= 64) GK_SCAN(8, 16);
        else if (d <= 128) GK_SCAN(16, 16);
        else if (d <= 256) GK_SCAN(32, 8);
        else GK_SCAN(64, 4);
    })
#undef GK_SCAN
    GK_CHECK_LAUNCH("memory_scan");
    return GK_OK;
}

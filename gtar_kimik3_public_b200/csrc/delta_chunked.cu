// The gated delta rule with one decay per head (see delta_head.cu) over many tokens at once, for bfloat16 steps: chunks of 64
// tokens whose inner work is matrix products that all chunks do side by side, and a walk over the chunks that carries the
// state in registers.
//
// Inside a chunk that starts from S0 let c_t = log g_0 + .. + log g_t (all exponents below are differences c_t - c_j with
// j <= t, so nothing grows), and let the unit vectors be k_t = a_t K_t, q_t = b_t Q_t with K_t, Q_t rounded to bfloat16 and 32-bit
// factors a_t, b_t.  The writes u_t solve a lower triangular system,
//     u_t = beta_t (v_t - e^(c_t) S0^T k_t - sum_{j<t} e^(c_t - c_j) (k_j . k_t) u_j)
// so with A_tj = beta_t e^(c_t - c_j) a_t a_j (K_t . K_j) below the diagonal and M = (1 + A)^-1 diag(beta)
//     u   = M (v - diag(e^c a) K S0)
//     o   = diag(e^c b) Q S0 + P u              P_tj = e^(c_t - c_j) b_t a_j (Q_t . K_j) for j <= t
//     S1  = e^(c_last) S0 + K^T diag(e^(c_last - c) a) u
// (the chunked form of the delta rule: S. Yang, B. Wang, Y. Zhang, Y. Shen, Y. Kim, "Parallelizing Linear Transformers with the
// Delta Rule over Sequence Length", and with decays S. Yang, J. Kautz, A. Hatamizadeh, "Gated Delta Networks: Improving Mamba2
// with Delta Rule".)
//
//   inner   a block per chunk and head: M, P and the factors of the chunk's tokens
//   walk    a block per head and 16 value columns, the chunks in sequence.  Four warps carry S^T in the accumulators of their
//           products (a quarter of the key entries each) and four form the read-outs beside them; what a product leaves for
//           the next one passes through shared memory, three barriers a chunk.  The next chunk's tiles are on their way
//           meanwhile.
//
// K, Q and V are bfloat16 numbers; every other operand (the state, v less its prediction, u, M, P) is a 32-bit number split into
// two bfloat16 halves, the rounded number and the rounded rest; what is left out is 2^-17 of a product.  Sums are 32-bit.

#include "attention_mma.cuh"

namespace {

using namespace attn;
typedef __nv_bfloat16 bf16;

constexpr int CHUNK = 64;
constexpr int INNER_THREADS = 128;
constexpr int LDA = CHUNK + 4;  // floats a row of A: 16-byte rows that start four banks apart
constexpr int TILE = CHUNK * CHUNK;

// What `inner` leaves for `walk`, per chunk and head: M (rounded, rest), P (rounded, rest), each a swizzled 64 x 64 tile, and the
// factors e^c a, e^c b, e^(c_last - c) a of the tokens and e^(c_last).
constexpr int WORK_BF16 = 4 * TILE;
constexpr int WORK_F32 = 3 * CHUNK + 4;

__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x, y);
    const float2 back = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
    lo = pack_bf16(x - back.x, y - back.y);
}

// 64 rows of d entries (a multiple of 8, at most D), `ld` apart, into a swizzled tile with rows of D; the rest is zero.
template <int D>
__device__ __forceinline__ void stage_rows(bf16* tile, const bf16* __restrict__ src, int ld, int valid, int d, int thread, int n_threads) {
    constexpr int PIECES = D / 8;
#pragma unroll 4
    for (int i = thread; i < CHUNK * PIECES; i += n_threads) {
        const int row = i / PIECES, piece = i % PIECES;
        const bool in = row < valid && piece * 8 < d;
        cp_async_16(reinterpret_cast<uint4*>(tile) + swz<D>(row, piece), src + (in ? row * ld + piece * 8 : 0), in);
    }
}

// Rows t0 .. t0+15 of X K^T (X, K swizzled tiles), the first `n_groups` groups of 16 columns.
template <int D>
__device__ __forceinline__ void rows_product(float (&s)[8][4], const bf16* x, const bf16* k, int t0, int n_groups, int lane) {
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) s[n][i] = 0.f;
    const int xrow = t0 + (lane & 7) + (((lane >> 3) & 1) << 3), krow = (lane & 7) + ((lane >> 4) << 3);
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t a[4];
        ldmatrix_x4(a, reinterpret_cast<const uint4*>(x) + swz<D>(xrow, ks * 2 + (lane >> 4)));
#pragma unroll
        for (int g = 0; g < 4; ++g) {
            if (g >= n_groups) continue;
            uint32_t b[4];
            ldmatrix_x4(b, reinterpret_cast<const uint4*>(k) + swz<D>(g * 16 + krow, ks * 2 + ((lane >> 3) & 1)));
            mma_16816(s[2 * g], a, b[0], b[1]);
            mma_16816(s[2 * g + 1], a, b[2], b[3]);
        }
    }
}

// a pair of neighbouring entries of a split tile (rounded half at `tile`, rest TILE behind)
__device__ __forceinline__ void store_split(bf16* tile, int row, int col, float x, float y) {
    uint32_t hi, lo;
    split2(x, y, hi, lo);
    const int at = swz<CHUNK>(row, col >> 3) * 8 + (col & 7);
    *reinterpret_cast<uint32_t*>(tile + at) = hi;
    *reinterpret_cast<uint32_t*>(tile + TILE + at) = lo;
}

template <int D>
__global__ void __launch_bounds__(INNER_THREADS) delta_inner_kernel(
    const bf16* __restrict__ q, const bf16* __restrict__ k, const float* __restrict__ q_unit, const float* __restrict__ k_unit,
    const float* __restrict__ log_g, const float* __restrict__ beta, bf16* __restrict__ work, float* __restrict__ factors,
    const int* __restrict__ cu_q, int n_heads, int n_kv, int d, int chunk0, int wave) {
    extern __shared__ __align__(128) unsigned char smem_raw[];
    bf16* qs = reinterpret_cast<bf16*>(smem_raw);             // [CHUNK][D]
    bf16* ks = qs + CHUNK * D;                                // [CHUNK][D]
    float* A = reinterpret_cast<float*>(ks + CHUNK * D);      // [CHUNK][LDA], below the diagonal
    __shared__ float c[CHUNK], a[CHUNK], b[CHUNK], bt[CHUNK];
    pdl_launch_dependents();
    const int in_wave = blockIdx.x, head = blockIdx.y, seq = blockIdx.z, hk = head / (n_heads / n_kv);
    pdl_wait();
    const int t0 = cu_q[seq], len = cu_q[seq + 1] - t0;
    const int first = (chunk0 + in_wave) * CHUNK;
    if (first >= len) return;
    const int n = min(CHUNK, len - first), tok0 = t0 + first;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    stage_rows<D>(qs, q + ((size_t)tok0 * n_kv + hk) * d, n_kv * d, n, d, tid, INNER_THREADS);
    stage_rows<D>(ks, k + ((size_t)tok0 * n_kv + hk) * d, n_kv * d, n, d, tid, INNER_THREADS);
    cp_async_commit();
    if (tid < CHUNK) {
        const bool in = tid < n;
        c[tid] = in ? log_g[(size_t)(tok0 + tid) * n_heads + head] : 0.f;
        bt[tid] = in ? beta[(size_t)(tok0 + tid) * n_heads + head] : 0.f;
        a[tid] = in ? k_unit[(size_t)(tok0 + tid) * n_kv + hk] : 0.f;
        b[tid] = in ? q_unit[(size_t)(tok0 + tid) * n_kv + hk] : 0.f;
    }
    __syncthreads();
    if (warp == 0) {  // running sums, two tokens a lane
        const float f0 = c[2 * lane], f1 = c[2 * lane + 1];
        float s = f0 + f1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += up;
        }
        c[2 * lane] = s - f1;
        c[2 * lane + 1] = s;
    }
    cp_async_wait<0>();
    __syncthreads();
    const size_t unit = ((size_t)seq * wave + in_wave) * n_heads + head;
    bf16* w = work + unit * WORK_BF16;
    float* f = factors + unit * WORK_F32;
    if (tid < CHUNK) {  // behind the chunk's end a is zero
        const float last = c[CHUNK - 1];
        f[tid] = expf(c[tid]) * a[tid];
        f[CHUNK + tid] = expf(c[tid]) * b[tid];
        f[2 * CHUNK + tid] = expf(last - c[tid]) * a[tid];
        if (tid == 0) f[3 * CHUNK] = expf(last);
    }
    // a warp has 16 tokens
    const int w0 = warp * 16;
    float s[8][4];
    rows_product<D>(s, ks, ks, w0, warp + 1, lane);
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int t = w0 + (lane >> 2) + 8 * (i >> 1), j = nt * 8 + (lane & 3) * 2 + (i & 1);
            A[t * LDA + j] = j < t ? bt[t] * expf(c[t] - c[j]) * (a[t] * a[j]) * s[nt][i] : 0.f;
        }
    rows_product<D>(s, qs, ks, w0, warp + 1, lane);
#pragma unroll
    for (int nt = 0; nt < 8; ++nt)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int t = w0 + (lane >> 2) + 8 * h, j = nt * 8 + (lane & 3) * 2;
            const float x = j <= t ? expf(c[t] - c[j]) * (b[t] * a[j]) * s[nt][2 * h] : 0.f;
            const float y = j + 1 <= t ? expf(c[t] - c[j + 1]) * (b[t] * a[j + 1]) * s[nt][2 * h + 1] : 0.f;
            store_split(w + 2 * TILE, t, j, x, y);
        }
    __syncthreads();
    // a column of (1 + A)^-1 a thread: x_i = [i = column] - sum_{j<i} A_ij x_j
    float x[CHUNK];
    if (tid < CHUNK) {
#pragma unroll
        for (int i = 0; i < CHUNK; ++i) {
            float p[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int j4 = 0; j4 < (i + 3) / 4; ++j4) {
                const float4 row = *reinterpret_cast<const float4*>(A + i * LDA + 4 * j4);
                const float e[4] = {row.x, row.y, row.z, row.w};
#pragma unroll
                for (int r = 0; r < 4; ++r)
                    if (4 * j4 + r < i) p[r] = fmaf(e[r], x[4 * j4 + r], p[r]);
            }
            x[i] = (i == tid ? 1.f : 0.f) - ((p[0] + p[1]) + (p[2] + p[3]));
        }
    }
    __syncthreads();
    if (tid < CHUNK) {
        const float mine = bt[tid];
#pragma unroll
        for (int i = 0; i < CHUNK; ++i) A[i * LDA + tid] = x[i] * mine;
    }
    __syncthreads();
    for (int i = tid; i < TILE / 2; i += INNER_THREADS) {
        const int row = i / (CHUNK / 2), col = (i % (CHUNK / 2)) * 2;
        store_split(w, row, col, A[row * LDA + col], A[row * LDA + col + 1]);
    }
}

constexpr int STRIP = 16;  // value columns of a block of the walk
constexpr int WALK_THREADS = 256;

template <int D>
struct WalkSmem {
    struct Stage {
        bf16 k[CHUNK * D], q[CHUNK * D];
        bf16 work[WORK_BF16];
        bf16 v[CHUNK * (STRIP + 8)];
        float factors[WORK_F32];
    } stage[2];
    // what the warps hand one another, each as a rounded half and a rest, rows of value columns
    bf16 state[2][STRIP][D + 8];          // S^T before the chunk
    bf16 rest[2][STRIP][CHUNK + 8];       // v less its prediction
    bf16 u[2][STRIP][CHUNK + 8];          // u
    bf16 scaled[2][STRIP][CHUNK + 8];     // u times e^(c_last - c) a
};

// the left operand's four registers for the 16 entries from k0 on
__device__ __forceinline__ void left_operand(uint32_t (&a)[4], const bf16* rows, int ld, int k0, int lane) {
    ldmatrix_x4(a, rows + ((lane & 7) + (((lane >> 3) & 1) << 3)) * ld + k0 + ((lane >> 4) << 3));
}

// Four warps (`walk`) carry the state, each a quarter of the key entries and 16 of a chunk's tokens; four more (`read`) form the
// read-outs of 16 tokens each beside them.
template <int D>
__global__ void __launch_bounds__(WALK_THREADS) delta_walk_kernel(
    const bf16* __restrict__ q, const bf16* __restrict__ k, const bf16* __restrict__ v, const bf16* __restrict__ work,
    const float* __restrict__ factors, float* __restrict__ state /* [slots, H, d, dv] */, float* __restrict__ out /* [T, H, dv] */,
    const int* __restrict__ cu_q, const int* __restrict__ slots, int n_heads, int n_kv, int d, int dv, int chunk0, int wave) {
    constexpr int V_LD = STRIP + 8, SD = D + 8, CD = CHUNK + 8, OWN = D / 4;
    extern __shared__ __align__(128) unsigned char smem_raw[];
    WalkSmem<D>& sm = *reinterpret_cast<WalkSmem<D>*>(smem_raw);
    pdl_launch_dependents();
    const int head = blockIdx.y, seq = blockIdx.z, hk = head / (n_heads / n_kv), v0 = blockIdx.x * STRIP;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, part = warp & 3;
    const bool walks = warp < 4;
    pdl_wait();
    const int t0 = cu_q[seq], len = cu_q[seq + 1] - t0;
    const int here = min(wave, (len + CHUNK - 1) / CHUNK - chunk0);
    if (here <= 0) return;
    // the tiles of chunk i, by n_threads threads of which this is the thread-th
    auto issue = [&](int i, int thread, int n_threads) {
        if (i < here) {
            auto& st = sm.stage[i & 1];
            const int first = (chunk0 + i) * CHUNK, n = min(CHUNK, len - first);
            const size_t tok0 = (size_t)(t0 + first);
            const size_t unit = ((size_t)seq * wave + i) * n_heads + head;
            stage_rows<D>(st.k, k + (tok0 * n_kv + hk) * d, n_kv * d, n, d, thread, n_threads);
            stage_rows<D>(st.q, q + (tok0 * n_kv + hk) * d, n_kv * d, n, d, thread, n_threads);
            const bf16* w = work + unit * WORK_BF16;
#pragma unroll 4
            for (int p = thread; p < WORK_BF16 / 8; p += n_threads) {
                const int row = (p >> 3) & (CHUNK - 1), piece = (p & 7) ^ (row & 7);  // M and P are lower triangular
                if (piece < 2 * (row / 16 + 1)) cp_async_16(st.work + p * 8, w + p * 8, true);
            }
            if (thread < WORK_F32 / 4) cp_async_16(st.factors + thread * 4, factors + unit * WORK_F32 + thread * 4, true);
            if (thread < CHUNK * 2) {
                const int row = thread >> 1, col = (thread & 1) * 8;
                const bool in = row < n && v0 + col < dv;
                cp_async_16(st.v + row * V_LD + col, v + (in ? (tok0 + row) * n_heads * dv + (size_t)head * dv + v0 + col : 0), in);
            }
        }
        cp_async_commit();
    };
    issue(0, threadIdx.x, WALK_THREADS);
    const int vrow = lane >> 2, pair = (lane & 3) * 2;                               // an accumulator's row and first column
    const int brow = (lane & 7) + ((lane >> 4) << 3), bpiece = (lane >> 3) & 1;      // operand rows of [n][k] tiles
    const int trow = (lane & 7) + (((lane >> 3) & 1) << 3), tpiece = lane >> 4;      // of [k][n] tiles, transposed on the way
    float* mine = state + ((size_t)slots[seq] * n_heads + head) * (size_t)d * dv;
    float S[OWN / 8][4];  // S^T: rows value columns, columns the warp's key entries
    auto publish_state = [&]() {
#pragma unroll
        for (int nt = 0; nt < OWN / 8; ++nt)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                uint32_t hi, lo;
                split2(S[nt][2 * h], S[nt][2 * h + 1], hi, lo);
                const int col = part * OWN + nt * 8 + pair;
                *reinterpret_cast<uint32_t*>(&sm.state[0][vrow + 8 * h][col]) = hi;
                *reinterpret_cast<uint32_t*>(&sm.state[1][vrow + 8 * h][col]) = lo;
            }
    };
    if (walks) {
#pragma unroll
        for (int nt = 0; nt < OWN / 8; ++nt)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int row = v0 + vrow + 8 * (i >> 1), col = part * OWN + nt * 8 + pair + (i & 1);
                S[nt][i] = row < dv && col < d ? mine[(size_t)col * dv + row] : 0.f;
            }
        publish_state();
    }
    const int tok = part * 16;  // the warp's tokens of a chunk
    for (int i = 0; i < here; ++i) {
        cp_async_wait<0>();
        __syncthreads();  // the chunk's tiles and the state before it are there; the other stage is free
        const auto& st = sm.stage[i & 1];
        // S0^T K^T (walk) or S0^T Q^T (read) for the warp's tokens; the two halves of the state add up on their own
        const bf16* rows = walks ? st.k : st.q;
        float acc[2][4], low[2][4];
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[nt][e] = low[nt][e] = 0.f;
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
            uint32_t hi[4], lo[4], b[4];
            left_operand(hi, &sm.state[0][0][0], SD, ks * 16, lane);
            left_operand(lo, &sm.state[1][0][0], SD, ks * 16, lane);
            ldmatrix_x4(b, reinterpret_cast<const uint4*>(rows) + swz<D>(tok + brow, ks * 2 + bpiece));
            mma_16816(acc[0], hi, b[0], b[1]);
            mma_16816(acc[1], hi, b[2], b[3]);
            mma_16816(low[0], lo, b[0], b[1]);
            mma_16816(low[1], lo, b[2], b[3]);
        }
        const float* f = st.factors + (walks ? 0 : CHUNK) + tok + pair;
        const float2 f0 = *reinterpret_cast<const float2*>(f), f1 = *reinterpret_cast<const float2*>(f + 8);
        const float fs[2][2] = {{f0.x, f0.y}, {f1.x, f1.y}};
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[nt][e] = (acc[nt][e] + low[nt][e]) * fs[nt][e & 1];
        if (walks) {  // v less its prediction
            uint32_t vt[4];  // transposed: (tokens 0-7, columns 0-7), (0-7, 8-15), (8-15, 0-7), (8-15, 8-15)
            ldmatrix_x4_trans(vt, st.v + (tok + (lane & 7) + ((lane >> 4) << 3)) * V_LD + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const float2 val = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&vt[2 * nt + h]));
                    uint32_t hi, lo;
                    split2(val.x - acc[nt][2 * h], val.y - acc[nt][2 * h + 1], hi, lo);
                    *reinterpret_cast<uint32_t*>(&sm.rest[0][vrow + 8 * h][tok + nt * 8 + pair]) = hi;
                    *reinterpret_cast<uint32_t*>(&sm.rest[1][vrow + 8 * h][tok + nt * 8 + pair]) = lo;
                }
        }
        __syncthreads();
        bf16(*u)[STRIP][CD] = sm.u;
        if (walks) {  // u of the warp's tokens: M is lower triangular
            float x[2][4], y[2][4];
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) x[nt][e] = y[nt][e] = 0.f;
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
                if (ks > part) break;
                uint32_t hi[4], lo[4], mh[4], ml[4];
                left_operand(hi, &sm.rest[0][0][0], CD, ks * 16, lane);
                left_operand(lo, &sm.rest[1][0][0], CD, ks * 16, lane);
                const int at = swz<CHUNK>(tok + brow, ks * 2 + bpiece);
                ldmatrix_x4(mh, reinterpret_cast<const uint4*>(st.work) + at);
                ldmatrix_x4(ml, reinterpret_cast<const uint4*>(st.work + TILE) + at);
                mma_16816(x[0], hi, mh[0], mh[1]);
                mma_16816(x[1], hi, mh[2], mh[3]);
                mma_16816(y[0], lo, mh[0], mh[1]);
                mma_16816(y[1], lo, mh[2], mh[3]);
                mma_16816(y[0], hi, ml[0], ml[1]);
                mma_16816(y[1], hi, ml[2], ml[3]);
            }
            const float2 e0 = *reinterpret_cast<const float2*>(st.factors + 2 * CHUNK + tok + pair);
            const float2 e1 = *reinterpret_cast<const float2*>(st.factors + 2 * CHUNK + tok + 8 + pair);
            const float es[2][2] = {{e0.x, e0.y}, {e1.x, e1.y}};
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int h = 0; h < 2; ++h) {
                    const float ux = x[nt][2 * h] + y[nt][2 * h], uy = x[nt][2 * h + 1] + y[nt][2 * h + 1];
                    const int row = vrow + 8 * h, col = tok + nt * 8 + pair;
                    uint32_t hi, lo;
                    split2(ux, uy, hi, lo);
                    *reinterpret_cast<uint32_t*>(&u[0][row][col]) = hi;
                    *reinterpret_cast<uint32_t*>(&u[1][row][col]) = lo;
                    split2(ux * es[nt][0], uy * es[nt][1], hi, lo);
                    *reinterpret_cast<uint32_t*>(&sm.scaled[0][row][col]) = hi;
                    *reinterpret_cast<uint32_t*>(&sm.scaled[1][row][col]) = lo;
                }
        } else {
            issue(i + 1, threadIdx.x - WALK_THREADS / 2, WALK_THREADS / 2);  // these warps have nothing else to do here
        }
        __syncthreads();
        if (walks) {  // the state behind the chunk
            const float g_last = st.factors[3 * CHUNK];
            float y[OWN / 8][4];
#pragma unroll
            for (int nt = 0; nt < OWN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    S[nt][e] *= g_last;
                    y[nt][e] = 0.f;
                }
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
                uint32_t hi[4], lo[4];
                left_operand(hi, &sm.scaled[0][0][0], CD, ks * 16, lane);
                left_operand(lo, &sm.scaled[1][0][0], CD, ks * 16, lane);
#pragma unroll
                for (int j = 0; j < OWN / 16; ++j) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, reinterpret_cast<const uint4*>(st.k) + swz<D>(ks * 16 + trow, part * (OWN / 8) + j * 2 + tpiece));
                    mma_16816(S[2 * j], hi, b[0], b[1]);
                    mma_16816(S[2 * j + 1], hi, b[2], b[3]);
                    mma_16816(y[2 * j], lo, b[0], b[1]);
                    mma_16816(y[2 * j + 1], lo, b[2], b[3]);
                }
            }
#pragma unroll
            for (int nt = 0; nt < OWN / 8; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[nt][e] += y[nt][e];
            publish_state();  // its readers of this chunk are behind two barriers
        } else {  // the read-outs' part from inside the chunk
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) low[nt][e] = 0.f;
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
                if (ks > part) break;
                uint32_t hi[4], lo[4], ph[4], pl[4];
                left_operand(hi, &u[0][0][0], CD, ks * 16, lane);
                left_operand(lo, &u[1][0][0], CD, ks * 16, lane);
                const int at = swz<CHUNK>(tok + brow, ks * 2 + bpiece);
                ldmatrix_x4(ph, reinterpret_cast<const uint4*>(st.work + 2 * TILE) + at);
                ldmatrix_x4(pl, reinterpret_cast<const uint4*>(st.work + 3 * TILE) + at);
                mma_16816(acc[0], hi, ph[0], ph[1]);
                mma_16816(acc[1], hi, ph[2], ph[3]);
                mma_16816(low[0], lo, ph[0], ph[1]);
                mma_16816(low[1], lo, ph[2], ph[3]);
                mma_16816(low[0], hi, pl[0], pl[1]);
                mma_16816(low[1], hi, pl[2], pl[3]);
            }
            const int first = (chunk0 + i) * CHUNK, n = min(CHUNK, len - first);
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = tok + nt * 8 + pair + (e & 1), row = v0 + vrow + 8 * (e >> 1);
                    if (t < n && row < dv) out[((size_t)(t0 + first + t) * n_heads + head) * dv + row] = acc[nt][e] + low[nt][e];
                }
        }
    }
    cp_async_wait<0>();
    if (walks) {
#pragma unroll
        for (int nt = 0; nt < OWN / 8; ++nt)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int row = v0 + vrow + 8 * (i >> 1), col = part * OWN + nt * 8 + pair + (i & 1);
                if (row < dv && col < d) mine[(size_t)col * dv + row] = S[nt][i];
            }
    }
}

}  // namespace

static bool chunked_fits(int d, int dv) { return d > 0 && d <= 128 && d % 8 == 0 && dv > 0 && dv % 8 == 0; }
GK_EXPORT int gk_delta_chunked_fits(int d, int dv) { return chunked_fits(d, dv); }
// Sizes of the workspaces per sequence, chunk of a wave and head: bfloat16 numbers and 32-bit numbers.
GK_EXPORT int gk_delta_chunked_work(int which) { return which == 0 ? WORK_BF16 : WORK_F32; }

// q, k [T, G, d], v [T, H, dv] bfloat16; q_unit, k_unit [T, G], log_g, beta [T, H], out [T, H, dv], state [slots, H, d, dv] 32-bit.
// max_len bounds the sequences' token counts in this step; `wave` chunks of every sequence are in flight at a time.
GK_EXPORT int gk_delta_chunked(const void* q, const void* k, const void* v, const float* q_unit, const float* k_unit, const float* log_g,
                               const float* beta, void* work, float* factors, float* state, float* out, const int* cu_q,
                               const int* slots, int n_seqs, int n_heads, int n_kv, int d, int dv, int max_len, int wave, void* stream) {
    GK_REQUIRE(n_heads > 0 && n_heads <= 65535 && n_kv > 0 && n_heads % n_kv == 0 && n_seqs >= 0 && n_seqs <= 65535, "delta_chunked: bad counts");
    GK_REQUIRE(chunked_fits(d, dv), "delta_chunked: heads of %d / %d do not fit (multiples of 8, keys up to 128)", d, dv);
    GK_REQUIRE(max_len >= 0 && wave > 0 && work != nullptr && factors != nullptr, "delta_chunked: bad sizes");
    GK_REQUIRE((((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)work | (uintptr_t)factors) & 15) == 0, "delta_chunked: rows must start on 16 bytes");
    if (n_seqs == 0 || max_len == 0) return GK_OK;
    static bool prepared = false;
    if (!prepared) {
#define GK_ATTR(KERNEL, BYTES)                                                                                                       \
    if (cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(BYTES)) != cudaSuccess) \
        return gk_fail(GK_CUDA_ERROR, "delta_chunked: shared memory")
        GK_ATTR((delta_inner_kernel<64>), 2 * CHUNK * 64 * 2 + CHUNK * LDA * 4);
        GK_ATTR((delta_inner_kernel<128>), 2 * CHUNK * 128 * 2 + CHUNK * LDA * 4);
        GK_ATTR((delta_walk_kernel<64>), sizeof(WalkSmem<64>));
        GK_ATTR((delta_walk_kernel<128>), sizeof(WalkSmem<128>));
#undef GK_ATTR
        prepared = true;
    }
    cudaStream_t s = (cudaStream_t)stream;
    const int chunks = (max_len + CHUNK - 1) / CHUNK, strips = (dv + STRIP - 1) / STRIP;
    for (int chunk0 = 0; chunk0 < chunks; chunk0 += wave) {
        const int here = chunks - chunk0 < wave ? chunks - chunk0 : wave;
#define GK_INNER(D)                                                                                                                \
    gk_launch(delta_inner_kernel<D>, dim3(here, n_heads, n_seqs), dim3(INNER_THREADS), (size_t)2 * CHUNK * D * 2 + CHUNK * LDA * 4, s, \
              (const bf16*)q, (const bf16*)k, q_unit, k_unit, log_g, beta, (bf16*)work, factors, cu_q, n_heads, n_kv, d, chunk0, wave)
#define GK_WALK(D)                                                                                                                 \
    gk_launch(delta_walk_kernel<D>, dim3(strips, n_heads, n_seqs), dim3(WALK_THREADS), sizeof(WalkSmem<D>), s, (const bf16*)q, (const bf16*)k, \
              (const bf16*)v, (const bf16*)work, (const float*)factors, state, out, cu_q, slots, n_heads, n_kv, d, dv, chunk0, wave)
        if (d <= 64) {
            GK_INNER(64);
            GK_WALK(64);
        } else {
            GK_INNER(128);
            GK_WALK(128);
        }
#undef GK_WALK
#undef GK_INNER
    }
    GK_CHECK_LAUNCH("delta_chunked");
    return GK_OK;
}

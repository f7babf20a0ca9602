// The recurrence of a matrix memory (see matrix_memory.cu) over many tokens at once, for bfloat16 steps: chunks of 64 tokens
// whose inner work is matrix products that all chunks do side by side, with one short pass over the chunks in sequence.
//
// Inside a chunk of n tokens (j, t count from 0) that starts from C0, n0 and the running maximum m0, with F_t = f_0 + .. + f_t,
// a_j = i_j - F_j and M_t = max(m0, a_0, .., a_t):
//     m_t   = F_t + M_t
//     num_t = e^(m0 - M_t) C0^T q_t + sum_{j<=t} e^(a_j - M_t) (q_t . k_j) v_j                   (read)
//     n . q = e^(m0 - M_t) n0 . q_t + sum_{j<=t} e^(a_j - M_t) (q_t . k_j)
//     L = sum_j e^(a_j - A) k_j v_j^T ,  A = max_j a_j ,  and the same with k alone for n        (local)
//     M = max(m0, A) ;  C1 = e^(m0 - M) C0 + e^(A - M) L ;  m1 = F_(n-1) + M                     (carry)
// No exponent is positive, so nothing grows.
//
// Three kernels a wave of chunks.  `local`: a block per chunk, head and 64 value columns.  `carry`: four entries of the state
// a thread, the wave's chunks in sequence; it leaves C0, n0 and m0 of every chunk where L and A were.  `read`: a block per
// chunk and head that holds all of the head's columns, so that the division, the norm of the head, the weight and the
// sigmoid gate happen in its output stage and the next product's operand is what it writes.
//
// The products run on the tensor cores with 32-bit sums and operands that carry 32-bit numbers: q, k and v are bfloat16 as
// they come from the projection, and the other operand of every product (the state, the weighted values, the weights of
// the chunk's own keys) is a 32-bit number split into two bfloat16 halves, the rounded number and the rounded rest, each
// multiplied by itself; what is left out is 2^-17 of the number.

#include "attention_mma.cuh"
#include "matrix_memory.cuh"

namespace {

using namespace attn;
using namespace memory;

typedef __nv_bfloat16 bf16;

constexpr int CHUNK = 64;
constexpr int PAD = 8;  // bfloat16 entries a row of a tile is longer: the eight rows of an ldmatrix start in different banks
constexpr int LOCAL_THREADS = 256, CARRY_THREADS = 256;

struct Work {
    float* states;   // [n_seqs, wave, H, d * dv + d]: L, then C0 (and behind it the same of n)
    float* scalars;  // [n_seqs, wave, H, 3]: A, F_(n-1), then m0
    float* start;    // [n_seqs, H]: the running maximum before the wave
};

struct Gates {
    float a[CHUNK];    // a_j; -inf behind the chunk's end
    float sum[CHUNK];  // F_j
};

// F and a of a chunk's tokens, by the block's first 64 threads and its first warp.  Ends with a barrier.
__device__ __forceinline__ void chunk_gates(Gates& g, const bf16* __restrict__ proj, long long ld, const Columns& at,
                                            const float* __restrict__ gate_bias, float cap, int head, int n_heads, int tok0, int n) {
    if (threadIdx.x < CHUNK) {
        const int j = threadIdx.x;
        float i = -INFINITY, f = 0.f;
        if (j < n) {
            const bf16* row = proj + (size_t)(tok0 + j) * ld;
            i = log_input_gate(to_float(row[at.i + head]) + gate_bias[head], cap);
            f = log_forget_gate(to_float(row[at.f + head]) + gate_bias[n_heads + head], cap);
        }
        g.a[j] = i;
        g.sum[j] = f;
    }
    __syncthreads();
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        const float f0 = g.sum[2 * lane], f1 = g.sum[2 * lane + 1];
        float s = f0 + f1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s += up;
        }
        const float F1 = s, F0 = s - f1;
        g.sum[2 * lane] = F0;
        g.sum[2 * lane + 1] = F1;
        g.a[2 * lane] -= F0;
        g.a[2 * lane + 1] -= F1;
    }
    __syncthreads();
}

__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(x, y);
    const float2 back = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
    lo = pack_bf16(x - back.x, y - back.y);
}

// `rows` rows of `width` entries (a multiple of 8) into a tile of rows of `stride`; rows at or behind `valid` become zero.
__device__ __forceinline__ void stage_rows(bf16* tile, int stride, const bf16* __restrict__ src, long long ld, int rows, int valid, int width) {
    const int pieces = width >> 3;
    for (int i = threadIdx.x; i < rows * pieces; i += blockDim.x) {
        const int r = i / pieces, c = (i - r * pieces) * 8;
        cp_async_16(tile + r * stride + c, src + (r < valid ? (size_t)r * ld + c : 0), r < valid);
    }
}

// ---- local: L of one chunk, 64 value columns a block
__global__ void __launch_bounds__(LOCAL_THREADS) memory_local_kernel(
    const bf16* __restrict__ proj, long long ld, Columns at, const float* __restrict__ gate_bias, float cap, float k_scale, Work work,
    const float* __restrict__ n_state, const int* __restrict__ cu_q, const int* __restrict__ slots, int n_heads, int d, int dv,
    int chunk0, int wave, int col_tiles) {
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ Gates g;
    __shared__ float weight[CHUNK];
    const int ks_ld = d + PAD;
    constexpr int VS_LD = 64 + PAD;
    bf16* ks = reinterpret_cast<bf16*>(smem);  // [CHUNK][d + PAD]
    bf16* vh = ks + CHUNK * ks_ld;             // [CHUNK][64 + PAD]: the weighted values, rounded; before that the values
    bf16* vl = vh + CHUNK * VS_LD;             // the rest
    pdl_launch_dependents();
    const int in_wave = blockIdx.x / col_tiles, tile = blockIdx.x - in_wave * col_tiles, c0 = tile * 64;
    const int head = blockIdx.y, seq = blockIdx.z;
    pdl_wait();
    const int t0 = cu_q[seq], len = cu_q[seq + 1] - t0;
    const int first = (chunk0 + in_wave) * CHUNK;
    if (first >= len) return;
    const int n = min(CHUNK, len - first), tok0 = t0 + first;
    const int cols = min(64, dv - c0);
    stage_rows(ks, ks_ld, proj + (size_t)tok0 * ld + at.k + head * d, ld, CHUNK, n, d);
    stage_rows(vh, VS_LD, proj + (size_t)tok0 * ld + at.v + head * dv + c0, ld, CHUNK, n, cols);
    cp_async_commit();
    chunk_gates(g, proj, ld, at, gate_bias, cap, head, n_heads, tok0, n);
    float largest = fmaxf(g.a[threadIdx.x & 31], g.a[32 + (threadIdx.x & 31)]);
    largest = warp_max(largest);
    if (threadIdx.x < CHUNK) weight[threadIdx.x] = expf(g.a[threadIdx.x] - largest) * k_scale;
    cp_async_wait<0>();
    __syncthreads();
    for (int i = threadIdx.x; i < CHUNK * 32; i += LOCAL_THREADS) {  // two columns a turn, in place
        const int j = i >> 5, c = (i & 31) * 2;
        uint32_t hi = 0, lo = 0;
        if (c < cols) {
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vh + j * VS_LD + c));
            split2(v.x * weight[j], v.y * weight[j], hi, lo);
        }
        *reinterpret_cast<uint32_t*>(vh + j * VS_LD + c) = hi;
        *reinterpret_cast<uint32_t*>(vl + j * VS_LD + c) = lo;
    }
    __syncthreads();
    const size_t item = ((size_t)seq * wave + in_wave) * n_heads + head;
    float* dst = work.states + item * (size_t)(d * dv + d);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int m0 = warp * 16; m0 < d; m0 += LOCAL_THREADS / 2) {
        float acc[8][4] = {};
        const int k_row = ((lane >> 4) << 3) + (lane & 7), k_col = m0 + ((lane >> 3) & 1) * 8;
        const int v_row = (lane & 7) + (((lane >> 3) & 1) << 3), v_col = (lane >> 4) * 8;
#pragma unroll
        for (int k0 = 0; k0 < CHUNK; k0 += 16) {
            uint32_t a[4];
            ldmatrix_x4_trans(a, ks + (k0 + k_row) * ks_ld + k_col);
#pragma unroll
            for (int nt = 0; nt < 4; ++nt) {
                uint32_t b[4];
                ldmatrix_x4_trans(b, vh + (k0 + v_row) * VS_LD + nt * 16 + v_col);
                mma_16816(acc[2 * nt], a, b[0], b[1]);
                mma_16816(acc[2 * nt + 1], a, b[2], b[3]);
                ldmatrix_x4_trans(b, vl + (k0 + v_row) * VS_LD + nt * 16 + v_col);
                mma_16816(acc[2 * nt], a, b[0], b[1]);
                mma_16816(acc[2 * nt + 1], a, b[2], b[3]);
            }
        }
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
            const int col = c0 + nt * 8 + (lane & 3) * 2;
            if (col < dv) {
                const int row = m0 + (lane >> 2);
                *reinterpret_cast<float2*>(dst + (size_t)row * dv + col) = make_float2(acc[nt][0], acc[nt][1]);
                *reinterpret_cast<float2*>(dst + (size_t)(row + 8) * dv + col) = make_float2(acc[nt][2], acc[nt][3]);
            }
        }
    }
    if (tile == 0) {
        for (int r = threadIdx.x; r < d; r += LOCAL_THREADS) {
            float s = 0.f;
#pragma unroll 8
            for (int j = 0; j < CHUNK; ++j) s = fmaf(weight[j], __bfloat162float(ks[j * ks_ld + r]), s);
            dst[(size_t)d * dv + r] = s;
        }
        if (threadIdx.x == 0) {
            float* sc = work.scalars + item * 3;
            sc[0] = largest;
            sc[1] = g.sum[n - 1];
            if (in_wave == 0) work.start[(size_t)seq * n_heads + head] = n_state[((size_t)slots[seq] * n_heads + head) * (d + 1) + d];
        }
    }
}

// ---- carry: the wave's chunks in sequence, four entries of the state (or of n) a thread
__global__ void __launch_bounds__(CARRY_THREADS) memory_carry_kernel(Work work, float* __restrict__ state, float* __restrict__ n_state,
                                                                     const int* __restrict__ cu_q, const int* __restrict__ slots,
                                                                     int n_heads, int d, int dv, int chunk0, int wave) {
    pdl_launch_dependents();
    const int e = blockIdx.x * CARRY_THREADS + threadIdx.x;
    const int head = blockIdx.y, seq = blockIdx.z;
    pdl_wait();
    const int len = cu_q[seq + 1] - cu_q[seq];
    const int here = min(wave, (len + CHUNK - 1) / CHUNK - chunk0);
    if (here <= 0) return;
    const int size4 = d * dv / 4, all4 = size4 + d / 4;
    const size_t slot_head = (size_t)slots[seq] * n_heads + head;
    float* own = state + slot_head * (size_t)(d + 1) * dv;
    float* own_n = n_state + slot_head * (d + 1);
    const size_t item0 = (size_t)seq * wave * n_heads + head;
    const bool busy = e < all4, is_n = e >= size4;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    if (busy && !is_n) s = reinterpret_cast<const float4*>(own)[e];
    if (busy && is_n) {
        const float* p = own_n + (e - size4) * 4;
        s = make_float4(p[0], p[1], p[2], p[3]);
    }
    float m = work.start[(size_t)seq * n_heads + head];
    float4* w = reinterpret_cast<float4*>(work.states + item0 * (size_t)(d * dv + d)) + (busy ? e : 0);
    float* sc = work.scalars + item0 * 3;
    const size_t step = (size_t)n_heads * all4;
    const bool keeper = blockIdx.x == 0 && threadIdx.x == 0;
    constexpr int AHEAD = 8;  // loads in flight: the chain itself is a few operations a chunk
    for (int c0 = 0; c0 < here; c0 += AHEAD) {
        float4 add[AHEAD];
        float top[AHEAD], total[AHEAD];
#pragma unroll
        for (int a = 0; a < AHEAD; ++a)
            if (c0 + a < here) {
                if (busy) add[a] = __ldcg(w + (size_t)a * step);
                top[a] = __ldcg(sc + (size_t)a * n_heads * 3);
                total[a] = __ldcg(sc + (size_t)a * n_heads * 3 + 1);
            }
#pragma unroll
        for (int a = 0; a < AHEAD; ++a) {
            if (c0 + a >= here) break;
            const float M = fmaxf(m, top[a]), keep = expf(m - M), in = expf(top[a] - M);
            if (busy) {
                __stcg(w + (size_t)a * step, s);
                s.x = fmaf(keep, s.x, in * add[a].x), s.y = fmaf(keep, s.y, in * add[a].y);
                s.z = fmaf(keep, s.z, in * add[a].z), s.w = fmaf(keep, s.w, in * add[a].w);
            }
            if (keeper) sc[(size_t)a * n_heads * 3 + 2] = m;
            m = total[a] + M;
        }
        w += (size_t)AHEAD * step;
        sc += (size_t)AHEAD * n_heads * 3;
    }
    if (busy && !is_n) reinterpret_cast<float4*>(own)[e] = s;
    if (busy && is_n) {
        float* p = own_n + (e - size4) * 4;
        p[0] = s.x, p[1] = s.y, p[2] = s.z, p[3] = s.w;
    }
    if (blockIdx.x == 0) {  // nothing reads these copies in this kernel
        for (int c = threadIdx.x; c < dv; c += CARRY_THREADS) own[(size_t)d * dv + c] = m;
        if (threadIdx.x == 0) own_n[d] = m;
    }
}

// ---- read: one chunk and head a block; four groups of 16 tokens times WN groups of CW value columns, a warp each
constexpr int S_ROWS = 16;  // rows of the state a stage

template <int WN, int CW>
struct ReadTile {
    static constexpr int THREADS = 128 * WN, DV = WN * CW, V_LD = DV + PAD;
    static size_t bytes(int d) { return ((size_t)2 * CHUNK * (d + PAD) + (size_t)CHUNK * V_LD + (size_t)4 * S_ROWS * V_LD) * sizeof(bf16); }
};

template <int WN, int CW>
__global__ void __launch_bounds__(ReadTile<WN, CW>::THREADS, WN == 2 ? 2 : 1) memory_read_kernel(
    const bf16* __restrict__ proj, long long ld, Columns at, int g_at, const float* __restrict__ gate_bias, float cap, float k_scale,
    Work work, const float* __restrict__ norm_w, float eps, bf16* __restrict__ y, const int* __restrict__ cu_q, int n_heads, int d,
    int dv, int chunk0, int wave) {
    using Tile = ReadTile<WN, CW>;
    constexpr int DV = Tile::DV, V_LD = Tile::V_LD, THREADS = Tile::THREADS, NT = CW / 8;
    constexpr int PIECES = S_ROWS * DV / 4 / THREADS;  // 16-byte pieces of a stage of the state a thread brings
    static_assert(S_ROWS * DV / 4 % THREADS == 0, "a stage is whole pieces");
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ Gates g;
    __shared__ float top[CHUNK], from_start[CHUNK], floor_at[CHUNK], qn[CHUNK], square[WN][CHUNK];
    const int q_ld = d + PAD;
    bf16* qs = reinterpret_cast<bf16*>(smem);  // [CHUNK][d + PAD]
    bf16* ks = qs + CHUNK * q_ld;              // [CHUNK][d + PAD]
    bf16* vs = ks + CHUNK * q_ld;              // [CHUNK][DV + PAD]
    bf16* sh = vs + CHUNK * V_LD;              // [2][2][S_ROWS][DV + PAD]: two stages of (rounded state, rest)
    pdl_launch_dependents();
    const int in_wave = blockIdx.x, head = blockIdx.y, seq = blockIdx.z;
    pdl_wait();
    const int t0 = cu_q[seq], len = cu_q[seq + 1] - t0;
    const int first = (chunk0 + in_wave) * CHUNK;
    if (first >= len) return;
    const int n = min(CHUNK, len - first), tok0 = t0 + first;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bf16* row0 = proj + (size_t)tok0 * ld;
    stage_rows(qs, q_ld, row0 + at.q + head * d, ld, CHUNK, n, d);
    stage_rows(ks, q_ld, row0 + at.k + head * d, ld, CHUNK, n, d);
    stage_rows(vs, V_LD, row0 + at.v + head * dv, ld, CHUNK, n, dv);
    cp_async_commit();
    if (dv < DV) {  // columns that do not exist: zero, for they take part in the products and in the norm's sum
        const int extra = (DV - dv) >> 3;
        for (int i = tid; i < CHUNK * extra; i += THREADS) {
            const int r = i / extra, c = dv + (i - r * extra) * 8;
            *reinterpret_cast<uint4*>(vs + r * V_LD + c) = make_uint4(0u, 0u, 0u, 0u);
        }
    }
    const size_t item = ((size_t)seq * wave + in_wave) * n_heads + head;
    const float* c0 = work.states + item * (size_t)(d * dv + d);
    const float m0 = __ldcg(work.scalars + item * 3 + 2);

    float4 ahead[PIECES];
    auto fetch = [&](int k0) {
#pragma unroll
        for (int p = 0; p < PIECES; ++p) {
            const int i = tid + p * THREADS, r = i / (DV / 4), c = (i % (DV / 4)) * 4;
            ahead[p] = c < dv ? __ldcg(reinterpret_cast<const float4*>(c0 + (size_t)(k0 + r) * dv + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    };
    auto put = [&](int buf) {
        bf16* hi = sh + buf * 2 * S_ROWS * V_LD;
        bf16* lo = hi + S_ROWS * V_LD;
#pragma unroll
        for (int p = 0; p < PIECES; ++p) {
            const int i = tid + p * THREADS, r = i / (DV / 4), c = (i % (DV / 4)) * 4;
            uint2 h, l;
            split2(ahead[p].x, ahead[p].y, h.x, l.x);
            split2(ahead[p].z, ahead[p].w, h.y, l.y);
            *reinterpret_cast<uint2*>(hi + r * V_LD + c) = h;
            *reinterpret_cast<uint2*>(lo + r * V_LD + c) = l;
        }
    };
    fetch(0);
    chunk_gates(g, proj, ld, at, gate_bias, cap, head, n_heads, tok0, n);
    if (warp == 0) {  // M_t: the largest of m0 and the a_j up to t
        const float a0 = g.a[2 * lane];
        float s = fmaxf(a0, g.a[2 * lane + 1]);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, s, o);
            if (lane >= o) s = fmaxf(s, up);
        }
        float before = __shfl_up_sync(0xffffffffu, s, 1);
        if (lane == 0) before = m0;
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            const int t = 2 * lane + h;
            const float M = fmaxf(m0, h == 0 ? fmaxf(before, a0) : s);
            top[t] = M;
            from_start[t] = expf(m0 - M);
            floor_at[t] = expf(-(g.sum[t] + M));
        }
    }
    put(0);
    cp_async_wait<0>();
    __syncthreads();
    // n0 . q of every token
    for (int t = warp; t < n; t += THREADS / 32) {
        float s = 0.f;
        for (int i = lane; i < d; i += 32) s = fmaf(__ldcg(c0 + (size_t)d * dv + i), __bfloat162float(qs[t * q_ld + i]), s);
        s = warp_sum(s);
        if (lane == 0) qn[t] = s;
    }
    const int rg = warp & 3, cg = warp >> 2;
    const int a_row = rg * 16 + (lane & 15), a_col = (lane >> 4) * 8;           // A fragments of q
    const int b_row = (lane & 7) + (((lane >> 3) & 1) << 3), b_col = cg * CW + (lane >> 4) * 8;  // B fragments of rows x columns
    float acc[NT][4];
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[nt][i] = 0.f;
    // C0^T q
    for (int k0 = 0, buf = 0; k0 < d; k0 += S_ROWS, buf ^= 1) {
        if (k0 + S_ROWS < d) fetch(k0 + S_ROWS);
        uint32_t a[4];
        ldmatrix_x4(a, qs + a_row * q_ld + k0 + a_col);
        const bf16* hi = sh + buf * 2 * S_ROWS * V_LD;
#pragma unroll
        for (int nt = 0; nt < NT / 2; ++nt) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, hi + b_row * V_LD + nt * 16 + b_col);
            mma_16816(acc[2 * nt], a, b[0], b[1]);
            mma_16816(acc[2 * nt + 1], a, b[2], b[3]);
            ldmatrix_x4_trans(b, hi + (S_ROWS + b_row) * V_LD + nt * 16 + b_col);
            mma_16816(acc[2 * nt], a, b[0], b[1]);
            mma_16816(acc[2 * nt + 1], a, b[2], b[3]);
        }
        if (k0 + S_ROWS < d) put(buf ^ 1);
        __syncthreads();
    }
    const int r0 = rg * 16 + (lane >> 2);
    float row_sum[2] = {0.f, 0.f};
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
            acc[nt][2 * h] *= from_start[r0 + 8 * h];
            acc[nt][2 * h + 1] *= from_start[r0 + 8 * h];
        }
    // the chunk's own keys, 16 at a time, up to the group's last token
    const int kb_row = (lane & 7) + ((lane >> 4) << 3), kb_col = ((lane >> 3) & 1) * 8;
    for (int grp = 0; grp <= rg; ++grp) {
        float s[2][4] = {};
        for (int k0 = 0; k0 < d; k0 += 16) {
            uint32_t a[4], b[4];
            ldmatrix_x4(a, qs + a_row * q_ld + k0 + a_col);
            ldmatrix_x4(b, ks + (grp * 16 + kb_row) * q_ld + k0 + kb_col);
            mma_16816(s[0], a, b[0], b[1]);
            mma_16816(s[1], a, b[2], b[3]);
        }
#pragma unroll
        for (int nt = 0; nt < 2; ++nt)
#pragma unroll
            for (int h = 0; h < 2; ++h)
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const int j = grp * 16 + nt * 8 + (lane & 3) * 2 + c, t = r0 + 8 * h;
                    const float w = j <= t ? s[nt][2 * h + c] * k_scale * expf(g.a[j] - top[t]) : 0.f;
                    s[nt][2 * h + c] = w;
                    row_sum[h] += w;
                }
        uint32_t ph[4], pl[4];
        split2(s[0][0], s[0][1], ph[0], pl[0]);
        split2(s[0][2], s[0][3], ph[1], pl[1]);
        split2(s[1][0], s[1][1], ph[2], pl[2]);
        split2(s[1][2], s[1][3], ph[3], pl[3]);
#pragma unroll
        for (int nt = 0; nt < NT / 2; ++nt) {
            uint32_t b[4];
            ldmatrix_x4_trans(b, vs + (grp * 16 + b_row) * V_LD + nt * 16 + b_col);
            mma_16816(acc[2 * nt], ph, b[0], b[1]);
            mma_16816(acc[2 * nt + 1], ph, b[2], b[3]);
            mma_16816(acc[2 * nt], pl, b[0], b[1]);
            mma_16816(acc[2 * nt + 1], pl, b[2], b[3]);
        }
    }
    // the division, the norm of the head, weight and gate
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        row_sum[h] += __shfl_xor_sync(0xffffffffu, row_sum[h], 1);
        row_sum[h] += __shfl_xor_sync(0xffffffffu, row_sum[h], 2);
        const int t = r0 + 8 * h;
        const float dot = fmaf(from_start[t], t < n ? qn[t] : 0.f, row_sum[h]);
        const float inv = 1.f / (fmaxf(fabsf(dot), floor_at[t]) + DEN_ADD);
        float ss = 0.f;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt)
#pragma unroll
            for (int c = 0; c < 2; ++c) {
                const float o = acc[nt][2 * h + c] * inv;
                acc[nt][2 * h + c] = o;
                ss = fmaf(o, o, ss);
            }
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        if ((lane & 3) == 0) square[cg][t] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        const int t = r0 + 8 * h;
        if (t >= n) continue;
        float ss = 0.f;
#pragma unroll
        for (int w = 0; w < WN; ++w) ss += square[w][t];
        const float r = 1.f / sqrtf(ss / (float)dv + eps);
        const bf16* gate = proj + (size_t)(tok0 + t) * ld + g_at + head * dv;
        bf16* out = y + (size_t)(tok0 + t) * n_heads * dv + head * dv;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
            const int col = cg * CW + nt * 8 + (lane & 3) * 2;
            if (col < dv) {
                const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gate + col));
                const float2 w = *reinterpret_cast<const float2*>(norm_w + head * dv + col);
                const float lo = acc[nt][2 * h] * r * w.x / (1.f + expf(-z.x)), hi = acc[nt][2 * h + 1] * r * w.y / (1.f + expf(-z.y));
                *reinterpret_cast<uint32_t*>(out + col) = pack_bf16(lo, hi);
            }
        }
    }
}

size_t local_smem(int d) { return ((size_t)CHUNK * (d + PAD) + 2 * CHUNK * (64 + PAD)) * sizeof(bf16); }

bool fits(int d, int dv) { return d > 0 && dv > 0 && d % 16 == 0 && dv % 16 == 0 && d <= 256 && dv <= 512; }

template <int WN, int CW>
int launch_read(const bf16* proj, long long ld, const Columns& at, int g_at, const float* gate_bias, float cap, float k_scale, Work work,
                const float* norm_w, float eps, bf16* y, const int* cu_q, int n_seqs, int n_heads, int d, int dv, int chunk0, int here,
                int wave, cudaStream_t s) {
    static bool prepared = false;
    if (!prepared) {
        cudaError_t err = cudaFuncSetAttribute(memory_read_kernel<WN, CW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 216 * 1024);
        if (err != cudaSuccess) return gk_fail(GK_CUDA_ERROR, "memory_chunked: %s", cudaGetErrorString(err));
        prepared = true;
    }
    using Tile = ReadTile<WN, CW>;
    gk_launch(memory_read_kernel<WN, CW>, dim3(here, n_heads, n_seqs), dim3(Tile::THREADS), Tile::bytes(d), s, proj, ld, at, g_at, gate_bias,
              cap, k_scale, work, norm_w, eps, y, cu_q, n_heads, d, dv, chunk0, wave);
    GK_CHECK_LAUNCH("memory_read");
    return GK_OK;
}

}  // namespace

// The recurrence, the heads' norm and the gate over the step's tokens of every sequence (bfloat16 rows of a packed projection);
// y [n_tokens, H dv].  `max_len` bounds the sequences' token counts; `states` holds n_seqs * wave * H * (d dv + d) floats,
// `scalars` n_seqs * wave * H * 3, `start` n_seqs * H; `wave` chunks of every sequence are in flight at a time.
GK_EXPORT int gk_memory_chunked(const void* proj, long long ld, int q_at, int k_at, int v_at, int g_at, int i_at, int f_at,
                                const float* gate_bias, float cap, float* state, float* n_state, const float* norm_w, float eps, void* y,
                                float* states, float* scalars, float* start, const int* cu_q, const int* slots, int n_seqs, int n_heads,
                                int d, int dv, int max_len, int wave, void* stream) {
    GK_REQUIRE(n_heads > 0 && n_heads <= 65535 && n_seqs >= 0 && n_seqs <= 65535, "memory_chunked: bad counts");
    GK_REQUIRE(fits(d, dv), "memory_chunked: heads of %d / %d do not fit (multiples of 16, up to 256 / 512)", d, dv);
    GK_REQUIRE(cap > 0.f && eps > 0.f && max_len >= 0 && wave > 0 && states && scalars && start, "memory_chunked: bad sizes");
    GK_REQUIRE(ld % 8 == 0 && q_at % 8 == 0 && k_at % 8 == 0 && v_at % 8 == 0 && g_at % 2 == 0 && reinterpret_cast<uintptr_t>(proj) % 16 == 0,
               "memory_chunked: rows and their parts must start on 16 bytes");
    if (n_seqs == 0 || max_len == 0) return GK_OK;
    static bool prepared = false;
    if (!prepared) {
        cudaFuncSetAttribute(memory_local_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024);
        prepared = true;
    }
    const Columns at = {q_at, k_at, v_at, i_at, f_at};
    const Work work = {states, scalars, start};
    const float k_scale = 1.f / sqrtf((float)d);
    const bf16* p = (const bf16*)proj;
    cudaStream_t s = (cudaStream_t)stream;
    const int chunks = (max_len + CHUNK - 1) / CHUNK, col_tiles = (dv + 63) / 64, all4 = (d * dv + d) / 4;
    for (int chunk0 = 0; chunk0 < chunks; chunk0 += wave) {
        const int here = chunks - chunk0 < wave ? chunks - chunk0 : wave;
        gk_launch(memory_local_kernel, dim3(here * col_tiles, n_heads, n_seqs), dim3(LOCAL_THREADS), local_smem(d), s, p, ld, at, gate_bias,
                  cap, k_scale, work, (const float*)n_state, cu_q, slots, n_heads, d, dv, chunk0, wave, col_tiles);
        gk_launch(memory_carry_kernel, dim3((all4 + CARRY_THREADS - 1) / CARRY_THREADS, n_heads, n_seqs), dim3(CARRY_THREADS), 0, s, work,
                  state, n_state, cu_q, slots, n_heads, d, dv, chunk0, wave);
        GK_CHECK_LAUNCH("memory_chunked");
        int status;
#define GK_READ(WN, CW)                                                                                                              \
    launch_read<WN, CW>(p, ld, at, g_at, gate_bias, cap, k_scale, work, norm_w, eps, (bf16*)y, cu_q, n_seqs, n_heads, d, dv, chunk0, here, \
                        wave, s)
        if (dv <= 64) status = GK_READ(2, 32);
        else if (dv <= 128) status = GK_READ(2, 64);
        else if (dv <= 256) status = GK_READ(2, 128);
        else status = GK_READ(4, 128);
#undef GK_READ
        if (status != GK_OK) return status;
    }
    return GK_OK;
}

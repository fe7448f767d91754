// A selective state space over prompts (Mamba-2, state-space duality), 64 tokens at a time on the tensor cores.  Per head,
// with dt_t = softplus(z_t + dt_bias), a_t = -exp(A_log) dt_t and the B and C of the head's group,
//
//     S_t = exp(a_t) S_(t-1) + dt_t B_t x_t^T          (S: [n, vd], float32, one per cache slot)
//     y_t = S_t^T C_t + D x_t
//
// which over a chunk of tokens, with c_i = a_1 + .. + a_i, is four products:
//
//     scores  G_ij = C_i . B_j                                        W_ij = exp(c_i - c_j) dt_j G_ij for j <= i, W_ii += D
//     inside  y_i += sum_j W_ij x_j
//     before  y_i += exp(c_i) S_0^T C_i
//     state   S    = exp(c_last) S_0 + sum_j exp(c_last - c_j) dt_j B_j x_j^T
//
// x, B and C are bfloat16 (the convolution's output), so the first product is exact up to its 32-bit sum; in the others the
// 32-bit factor (W, S, the weighted x) enters as a sum of bfloat16 terms: three (all 24 bits of mantissa) for the weighted x,
// whose sums are carried on in S, two (16 bits) for W and the S that is read out, which reach one output each.  The sums c run in 64-bit and are kept as two floats, so that a difference of two of them is right
// to 32-bit rounding however long the sum is; no quotient of decays is ever formed.
//
// A block owns one head's state columns v0 .. v0 + VT - 1, a warp 16 of them, and keeps S^T in the accumulator registers of its
// mma tiles for the whole walk: the accumulator layout of S^T [16 x n] is the layout of the left operand of the "before"
// product, so the state never passes shared memory.  B, C and x of the next chunk arrive by asynchronous copies while a
// chunk is worked on.
//
// Long prompts of few sequences are cut into segments that run side by side: STATES gives every segment's own contribution to
// the state (from zero) and the product of its decays, `segment_starts_kernel` joins them, S before segment s + 1 = decays
// of s x S before segment s + contribution of s, and OUTPUTS walks every segment from its start; the last one leaves the
// sequence's state.  WHOLE walks a sequence's new tokens from and to its state in one go.
//
// Compiled for one pair of sizes: -DQ3_STATE=<n> -DQ3_VALUE_DIM=<vd>, multiples of 16 up to 256.
#include "common.cuh"

#if !defined(Q3_STATE) || !defined(Q3_VALUE_DIM)
#error "compile with -DQ3_STATE=<rows of the state> -DQ3_VALUE_DIM=<columns>"
#endif

namespace {

constexpr int NS = Q3_STATE, VD = Q3_VALUE_DIM;
static_assert(NS % 16 == 0 && NS >= 16 && NS <= 256 && VD % 16 == 0 && VD >= 16 && VD <= 256, "sizes: multiples of 16 up to 256");
constexpr int VT = VD % 64 == 0 ? 64 : (VD % 48 == 0 ? 48 : (VD % 32 == 0 ? 32 : 16));   // state columns a block
constexpr int WARPS = VT / 16, THREADS = WARPS * 32;
constexpr int C = 64;                                    // tokens of a chunk
constexpr int N_ROW = NS * 2 + 16, X_ROW = VT * 2 + 16, W_ROW = C * 2 + 16;   // bytes of padded rows: conflict-free ldmatrix
constexpr int N_TILE = C * N_ROW, X_TILE = C * X_ROW, W_TILE = C * W_ROW;
constexpr int STAGE = 2 * N_TILE + X_TILE;               // C, B, x of a chunk
constexpr int SMEM = 2 * STAGE + 2 * W_TILE;
static_assert(SMEM <= 226 * 1024, "the chunk's tiles have to fit an SM's shared memory");

enum Walk { WHOLE, STATES, OUTPUTS };

struct Args {
    const bf16* x;               // columns of rows `row` values apart: x head by head, B and C group by group
    const bf16* B;
    const bf16* C;
    int64_t row;
    const float* z;              // [tokens, H] step logits
    const float* dt_bias;        // [H]
    const float* a_log;
    const float* skip;
    float* state;                // slot s, head h at state + s * slot_stride + h * NS * VD
    int64_t slot_stride;
    const int* seq_start;
    const int* seq_slots;
    float* out;                  // [tokens, H, VD]
    int H, share;
    float* seg_states;           // [sequences, count, H, NS, VD], then [sequences, count, H] products of decays
    float* seg_decay;
    int seg_length, seg_count;
};

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
// 16 bytes, or zeros with `live` false (the source is then not read)
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool live) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(live ? 16 : 0));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int K> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(K)); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two values as pairs of bfloat16 terms: hi, what its rounding dropped, and what that rounding dropped.
__device__ __forceinline__ uint32_t take_term(float& a, float& b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    a -= __low2float(h);
    b -= __high2float(h);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float softplus_f32(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

template <Walk WALK>
__global__ void __launch_bounds__(THREADS)
ssd_kernel(const Args p) {
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float dt_s[C], hi_s[C], lo_s[C];          // step sizes; c_i = hi + lo
    pdl_launch_dependents();
    pdl_wait();
    const int head = blockIdx.x, seq = blockIdx.y, group = head / p.share;
    constexpr int COL_TILES = VD / VT;
    const int segment = WALK == WHOLE ? 0 : (int)blockIdx.z / COL_TILES;
    const int v0 = (int)(blockIdx.z - segment * COL_TILES) * VT;
    const int seq_end = p.seq_start[seq + 1], t_begin = p.seq_start[seq] + (WALK == WHOLE ? 0 : segment * p.seg_length);
    const int t_end = WALK == WHOLE ? seq_end : min(seq_end, t_begin + p.seg_length);
    if (t_begin >= seq_end) return;
    if (WALK == STATES && t_end == seq_end) return;      // the last segment's walk leaves the state itself
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int64_t per_head = (int64_t)NS * VD;
    float* S_g = p.state + (int64_t)p.seq_slots[seq] * p.slot_stride + head * per_head;
    float* S_seg = WALK == WHOLE ? nullptr : p.seg_states + (((int64_t)seq * p.seg_count + segment) * p.H + head) * per_head;

    // S^T: tile k holds state rows 8 k + 2 t, + 1 (columns of the tile) and state columns v0 + 16 warp + g, + 8
    float S[NS / 8][4];
    const int v_lane = v0 + warp * 16 + g;
    {
        const float* from = WALK == WHOLE ? S_g : S_seg;
#pragma unroll
        for (int k = 0; k < NS / 8; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e)
                S[k][e] = WALK == STATES ? 0.0f : from[(int64_t)(8 * k + 2 * t + (e & 1)) * VD + v_lane + (e >> 1) * 8];
    }
    const float rate = -expf(p.a_log[head]), dt_bias = p.dt_bias[head], skip = p.skip[head];
    const uint32_t base = smem_u32(smem), w_hi = base + 2 * STAGE, w_lo = w_hi + W_TILE;
    const bf16* x_g = p.x + (int64_t)head * VD + v0;
    const bf16* B_g = p.B + (int64_t)group * NS;
    const bf16* C_g = p.C + (int64_t)group * NS;

    auto issue = [&](int t0, int buffer) {               // the chunk from t0 on, rows beyond the walk as zeros
        if (t0 < t_end) {
            const uint32_t to = base + buffer * STAGE;
            constexpr int PER_N = NS / 8, PER_X = VT / 8;
            for (int i = tid; i < C * PER_N; i += THREADS) {
                const int r = i / PER_N, c = i % PER_N;
                const bool live = t0 + r < t_end;
                const int64_t at = (int64_t)(live ? t0 + r : t0) * p.row + c * 8;
                if (WALK != STATES) cp_async16(to + r * N_ROW + c * 16, C_g + at, live);
                cp_async16(to + N_TILE + r * N_ROW + c * 16, B_g + at, live);
            }
            for (int i = tid; i < C * PER_X; i += THREADS) {
                const int r = i / PER_X, c = i % PER_X;
                const bool live = t0 + r < t_end;
                cp_async16(to + 2 * N_TILE + r * X_ROW + c * 16, x_g + (int64_t)(live ? t0 + r : t0) * p.row + c * 8, live);
            }
        }
        cp_async_commit();
    };
    auto logit = [&](int t0, int i) { return t0 + i < t_end ? p.z[(int64_t)(t0 + i) * p.H + head] : 0.0f; };

    double total = 0.0;                                  // warp 0: c summed over the segment so far
    float z0 = 0.0f, z1 = 0.0f;
    issue(t_begin, 0);
    if (warp == 0) {
        z0 = logit(t_begin, 2 * lane);
        z1 = logit(t_begin, 2 * lane + 1);
    }
    // the rows of 8 x 8 matrices that this lane's address stands for: left operands / right operands as stored, transposed
    const int krow = (lane & 7) + ((lane >> 4) << 3), kcol = (lane >> 3) & 1;
    const int vrow = (lane & 7) + (((lane >> 3) & 1) << 3), vcol = lane >> 4;
    int buffer = 0;
    for (int t0 = t_begin; t0 < t_end; t0 += C, buffer ^= 1) {
        if (warp == 0) {                                 // steps and running sums of this chunk, two tokens a lane
            const int i = 2 * lane;
            const float d0 = t0 + i < t_end ? softplus_f32(z0 + dt_bias) : 0.0f, d1 = t0 + i + 1 < t_end ? softplus_f32(z1 + dt_bias) : 0.0f;
            const double a0 = (double)(rate * d0), a1 = (double)(rate * d1);
            double sum = a0 + a1;
#pragma unroll
            for (int off = 1; off < 32; off <<= 1) {
                const double before = __shfl_up_sync(0xffffffffu, sum, off);
                if (lane >= off) sum += before;
            }
            total += __shfl_sync(0xffffffffu, sum, 31);
            z0 = logit(t0 + C, i);                       // on their way for the next chunk
            z1 = logit(t0 + C, i + 1);
            __syncwarp();
            const double c1 = sum, c0 = sum - a1;
            // (nobody reads these of the chunk before any more: its last reads come before the barrier behind its weights,
            // or, where there are none, before the one at its end)
            dt_s[i] = d0; dt_s[i + 1] = d1;
            hi_s[i] = (float)c0; lo_s[i] = (float)(c0 - (double)(float)c0);
            hi_s[i + 1] = (float)c1; lo_s[i + 1] = (float)(c1 - (double)(float)c1);
        }
        cp_async_wait<0>();
        __syncthreads();                                 // the chunk has landed; every warp is done with the one before
        issue(t0 + C, buffer ^ 1);
        const uint32_t c_s = base + buffer * STAGE, b_s = c_s + N_TILE, x_s = b_s + N_TILE;
        const float hi_last = hi_s[C - 1], lo_last = lo_s[C - 1];
        if constexpr (WALK != STATES) {
            // scores: 16 rows of tokens i at a time, the blocks of 16 tokens j up to them; weighted and split into shared memory
            for (int mi = warp; mi < C / 16; mi += WARPS) {
                float s[C / 8][4];
#pragma unroll
                for (int j = 0; j < C / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.0f;
#pragma unroll
                for (int kt = 0; kt < NS / 16; ++kt) {
                    uint32_t a[4];
                    ldmatrix_x4(a, c_s + (mi * 16 + (lane & 15)) * N_ROW + (2 * kt + (lane >> 4)) * 16);
#pragma unroll
                    for (int jb = 0; jb < C / 16; ++jb) {
                        if (jb > mi) continue;
                        uint32_t b[4];
                        ldmatrix_x4(b, b_s + (jb * 16 + krow) * N_ROW + (2 * kt + kcol) * 16);
                        mma_bf16(s[2 * jb], a, b[0], b[1]);
                        mma_bf16(s[2 * jb + 1], a, b[2], b[3]);
                    }
                }
                const int i0 = mi * 16 + g;
                const float hi_i[2] = {hi_s[i0], hi_s[i0 + 8]}, lo_i[2] = {lo_s[i0], lo_s[i0 + 8]};
#pragma unroll
                for (int jt = 0; jt < C / 8; ++jt) {
                    if (jt > 2 * mi + 1) continue;
                    const int j = jt * 8 + 2 * t;
                    const float2 hj = *reinterpret_cast<const float2*>(hi_s + j), lj = *reinterpret_cast<const float2*>(lo_s + j);
                    const float2 dj = *reinterpret_cast<const float2*>(dt_s + j);
#pragma unroll
                    for (int r = 0; r < 2; ++r) {
                        const int i = i0 + 8 * r;
                        float w0 = j <= i ? s[jt][2 * r] * dj.x * expf((hi_i[r] - hj.x) + (lo_i[r] - lj.x)) : 0.0f;
                        float w1 = j + 1 <= i ? s[jt][2 * r + 1] * dj.y * expf((hi_i[r] - hj.y) + (lo_i[r] - lj.y)) : 0.0f;
                        if (j == i) w0 += skip;
                        if (j + 1 == i) w1 += skip;
                        const uint32_t at = i * W_ROW + j * 2, hi = take_term(w0, w1), lo = take_term(w0, w1);
                        asm volatile("st.shared.b32 [%0], %1;" ::"r"(w_hi + at), "r"(hi) : "memory");
                        asm volatile("st.shared.b32 [%0], %1;" ::"r"(w_lo + at), "r"(lo) : "memory");
                    }
                }
            }
        }
        // x^T of this warp's columns, 16 tokens a tile
        uint32_t xa[C / 16][4];
#pragma unroll
        for (int kt = 0; kt < C / 16; ++kt)
            ldmatrix_x4_trans(xa[kt], x_s + (kt * 16 + krow) * X_ROW + (warp * 2 + kcol) * 16);
        float keep_w[C / 16][4];                         // exp(c_last - c_j) dt_j of the tokens of this lane's fragments
#pragma unroll
        for (int kt = 0; kt < C / 16; ++kt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int j = kt * 16 + 2 * t + (e & 1) + (e >> 1) * 8;
                keep_w[kt][e] = dt_s[j] * expf((hi_last - hi_s[j]) + (lo_last - lo_s[j]));
            }
        const float keep_all = expf(hi_last + lo_last);
        if constexpr (WALK != STATES) {
            float before[C / 8][2];                      // exp(c_i) of this lane's output columns
#pragma unroll
            for (int it = 0; it < C / 8; ++it)
#pragma unroll
                for (int e = 0; e < 2; ++e) before[it][e] = expf(hi_s[it * 8 + 2 * t + e] + lo_s[it * 8 + 2 * t + e]);
            __syncthreads();                             // the weights are in place
            float y[C / 8][4];                           // y^T: rows are state columns, columns are tokens
#pragma unroll
            for (int it = 0; it < C / 8; ++it) y[it][0] = y[it][1] = y[it][2] = y[it][3] = 0.0f;
#pragma unroll
            for (int kt = 0; kt < NS / 16; ++kt) {
                // the accumulators of state rows 16 kt .. + 15 are a left operand as they lie
                float r[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) r[e] = S[2 * kt + (e >> 2)][e & 3];
                uint32_t s0[4], s1[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    s0[e] = take_term(r[2 * e], r[2 * e + 1]);
                    s1[e] = take_term(r[2 * e], r[2 * e + 1]);
                }
                uint32_t b[C / 16][4];
#pragma unroll
                for (int ib = 0; ib < C / 16; ++ib) ldmatrix_x4(b[ib], c_s + (ib * 16 + krow) * N_ROW + (2 * kt + kcol) * 16);
                // term by term over all the tiles: the products of one accumulator do not wait for one another back to back
#pragma unroll
                for (int it = 0; it < C / 8; ++it) mma_bf16(y[it], s1, b[it >> 1][2 * (it & 1)], b[it >> 1][2 * (it & 1) + 1]);
#pragma unroll
                for (int it = 0; it < C / 8; ++it) mma_bf16(y[it], s0, b[it >> 1][2 * (it & 1)], b[it >> 1][2 * (it & 1) + 1]);
            }
#pragma unroll
            for (int it = 0; it < C / 8; ++it)
#pragma unroll
                for (int e = 0; e < 4; ++e) y[it][e] *= before[it][e & 1];
#pragma unroll
            for (int kt = 0; kt < C / 16; ++kt) {
#pragma unroll
                for (int term = 1; term >= 0; --term) {
#pragma unroll
                    for (int ib = kt; ib < C / 16; ++ib) {
                        uint32_t b[4];
                        ldmatrix_x4(b, (term ? w_lo : w_hi) + (ib * 16 + krow) * W_ROW + (2 * kt + kcol) * 16);
                        mma_bf16(y[2 * ib], xa[kt], b[0], b[1]);
                        mma_bf16(y[2 * ib + 1], xa[kt], b[2], b[3]);
                    }
                }
            }
            float* out = p.out + ((int64_t)t0 * p.H + head) * VD + v_lane;
#pragma unroll
            for (int it = 0; it < C / 8; ++it)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int i = it * 8 + 2 * t + (e & 1);
                    if (t0 + i < t_end) out[(int64_t)i * p.H * VD + (e >> 1) * 8] = y[it][e];
                }
        }
        // the state after the chunk: S^T <- exp(c_last) S^T + (weighted x)^T B
#pragma unroll
        for (int k = 0; k < NS / 8; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) S[k][e] *= keep_all;
#pragma unroll
        for (int kt = 0; kt < C / 16; ++kt) {
            uint32_t x0[4], x1[4], x2[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {                // registers: (g, 2t), (g + 8, 2t), (g, 2t + 8), (g + 8, 2t + 8) and their neighbours
                const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(&xa[kt][e]);
                float a = __low2float(v) * keep_w[kt][(e >> 1) * 2], b = __high2float(v) * keep_w[kt][(e >> 1) * 2 + 1];
                x0[e] = take_term(a, b);
                x1[e] = take_term(a, b);
                x2[e] = take_term(a, b);
            }
            constexpr int NB = NS / 16 % 4 == 0 ? 4 : (NS / 16 % 2 == 0 ? 2 : 1);    // 16-row blocks of B at a time
#pragma unroll
            for (int nb = 0; nb < NS / 16; nb += NB) {
                uint32_t b[NB][4];
#pragma unroll
                for (int i = 0; i < NB; ++i) ldmatrix_x4_trans(b[i], b_s + (kt * 16 + vrow) * N_ROW + (2 * (nb + i) + vcol) * 16);
#pragma unroll
                for (int i = 0; i < 2 * NB; ++i) mma_bf16(S[2 * nb + i], x2, b[i >> 1][2 * (i & 1)], b[i >> 1][2 * (i & 1) + 1]);
#pragma unroll
                for (int i = 0; i < 2 * NB; ++i) mma_bf16(S[2 * nb + i], x1, b[i >> 1][2 * (i & 1)], b[i >> 1][2 * (i & 1) + 1]);
#pragma unroll
                for (int i = 0; i < 2 * NB; ++i) mma_bf16(S[2 * nb + i], x0, b[i >> 1][2 * (i & 1)], b[i >> 1][2 * (i & 1) + 1]);
            }
        }
        if constexpr (WALK == STATES) __syncthreads();   // the sums and steps may be rewritten
    }
    cp_async_wait<0>();
    if (WALK == STATES && tid == 0 && v0 == 0)
        p.seg_decay[((int64_t)seq * p.seg_count + segment) * p.H + head] = (float)exp(total);
    if (WALK == OUTPUTS && t_end < seq_end) return;
    float* to = WALK == STATES ? S_seg : S_g;
#pragma unroll
    for (int k = 0; k < NS / 8; ++k)
#pragma unroll
        for (int e = 0; e < 4; ++e) to[(int64_t)(8 * k + 2 * t + (e & 1)) * VD + v_lane + (e >> 1) * 8] = S[k][e];
}

// A thread per value of a sequence's state: the contributions of its segments become the states before them.
__global__ void segment_starts_kernel(const Args p) {
    pdl_launch_dependents();
    pdl_wait();
    const int seq = blockIdx.y;
    const int64_t x = (int64_t)blockIdx.x * blockDim.x + threadIdx.x, per_head = (int64_t)NS * VD, all = p.H * per_head;
    if (x >= all) return;
    const int live = (p.seq_start[seq + 1] - p.seq_start[seq] + p.seg_length - 1) / p.seg_length;
    const float* decay = p.seg_decay + (int64_t)seq * p.seg_count * p.H + x / per_head;
    float S = p.state[(int64_t)p.seq_slots[seq] * p.slot_stride + x];
    float* at = p.seg_states + (int64_t)seq * p.seg_count * all + x;
    for (int s0 = 0; s0 < live; s0 += 8, at += 8 * all) {
        float own[8], keep[8];                           // eight loads on their way together
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            own[i] = s0 + i + 1 < live ? at[i * all] : 0.0f;
            keep[i] = s0 + i + 1 < live ? decay[(int64_t)(s0 + i) * p.H] : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (s0 + i < live) at[i * all] = S;
            S = fmaf(keep[i], S, own[i]);
        }
    }
}

// The number of segments (1: none) for prompts of at most `max_new` tokens: as many blocks as run at once, two per multiprocessor
// (one block more and the last of them run alone: one prompt of 2,048 tokens with 128 heads took 226 us in 2 segments, 274 in 3),
// segments of at least two chunks, at most 64 MB of states.
int segment_count(int n_seqs, int max_new, int H) {
    const int64_t blocks = (int64_t)H * n_seqs * (VD / VT), bytes = (int64_t)n_seqs * H * NS * VD * 4;
    const int64_t want = 2 * (int64_t)q3_device_sm_count() / blocks;
    int64_t count = want < max_new / (2 * C) ? want : max_new / (2 * C);
    if (count > (64ll << 20) / bytes) count = (64ll << 20) / bytes;
    return count < 2 ? 1 : (int)count;
}

int ssd_launch(Args p, int n_seqs, float* scratch, int max_new, int count, cudaStream_t stream) {
    if (n_seqs <= 0 || max_new <= 0) return 0;
    if (p.H <= 0 || p.share <= 0 || p.H % p.share != 0 || n_seqs > 65535 || p.row % 8 != 0) return Q3_ERR_BAD_SIZE;
    if (!aligned16(p.x) || !aligned16(p.B) || !aligned16(p.C)) return Q3_ERR_MISALIGNED;
    if (scratch == nullptr || count < 1) count = 1;
    static Q3PerDevice allowed[3];
    auto walk = [&](auto kernel, Q3PerDevice& done, int segments) {
        const cudaError_t e = q3_allow_shared_memory(kernel, SMEM, done);
        if (e != cudaSuccess) return (int)e;
        return (int)q3_launch(kernel, dim3(p.H, n_seqs, VD / VT * segments), dim3(THREADS), SMEM, stream, p);
    };
    p.seg_states = p.seg_decay = nullptr;
    p.seg_length = 0;
    p.seg_count = 1;
    if (count == 1) return walk(ssd_kernel<WHOLE>, allowed[0], 1);
    p.seg_length = ((max_new + count - 1) / count + C - 1) / C * C;
    p.seg_count = count;
    p.seg_states = scratch;
    p.seg_decay = scratch + (int64_t)n_seqs * count * p.H * NS * VD;
    if ((int64_t)p.seg_length * count < max_new || (int64_t)(VD / VT) * count > 65535) return Q3_ERR_BAD_SIZE;
    int code = walk(ssd_kernel<STATES>, allowed[1], count - 1);
    if (code != 0) return code;
    const int64_t all = (int64_t)p.H * NS * VD;
    code = (int)q3_launch(segment_starts_kernel, dim3((unsigned)((all + 255) / 256), n_seqs), dim3(256), 0, stream, p);
    if (code != 0) return code;
    return walk(ssd_kernel<OUTPUTS>, allowed[2], count);
}

}  // namespace

// x [tokens, H * VD], B and C [tokens, H / share * NS]: columns of rows `row` values apart; z float32 [tokens, H]; out float32
// [tokens, H * VD].  `segments` > 1: `scratch` holds n_seqs * segments * H * (NS * VD + 1) float32.
Q3_EXPORT int q3_ssd_prompt_bf16(const void* x, const void* B, const void* C_rows, int64_t row, const float* z, const float* dt_bias,
                                 const float* a_log, const float* skip, float* state, int64_t slot_stride, const int* seq_start,
                                 const int* seq_slots, float* out, int n_seqs, int heads, int share, float* scratch, int max_new,
                                 int segments, void* stream) {
    Args p;
    p.x = (const bf16*)x; p.B = (const bf16*)B; p.C = (const bf16*)C_rows; p.row = row; p.z = z; p.dt_bias = dt_bias; p.a_log = a_log;
    p.skip = skip; p.state = state; p.slot_stride = slot_stride; p.seq_start = seq_start; p.seq_slots = seq_slots; p.out = out;
    p.H = heads; p.share = share;
    return ssd_launch(p, n_seqs, scratch, max_new, segments, (cudaStream_t)stream);
}
Q3_EXPORT int q3_ssd_segments(int n_seqs, int max_new, int heads) {
    if (n_seqs <= 0 || max_new <= 0 || heads <= 0) return 1;
    return segment_count(n_seqs, max_new, heads);
}

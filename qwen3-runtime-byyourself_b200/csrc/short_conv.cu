// A short causal convolution over time on every channel of a projection's rows, with the last taps - 1 input rows of
// every sequence kept as its state:
//
//     y[t, c] = sum_j w[c, j] * u[t - taps + 1 + j, c],   j = 0 .. taps - 1,   u = 0 before the sequence's start
//
// With `bias` a number per channel is added to the sum, with `silu` the result goes through SiLU, all before the rounding.
//
//   short_conv       : one thread per (token, channel) - or, for 2 to 4 taps and rows of 16-byte packets, per run of up to 16
//                      tokens and packet of channels, the last rows kept in registers; an input row before the step's first
//                      token comes from the state [slot][taps - 1][C] (float32; the oldest row first), zeros for a new sequence.
//                      The products are summed in 32-bit in ascending j whatever the step, so a token's output is the
//                      same bits however the sequence was cut.
//   short_conv_step  : steps of one token per sequence: a thread per (sequence, packet of channels) does both at once.
//   short_conv_state : afterwards, one thread per (sequence, channel) moves the state on: the last taps - 1 rows of
//                      (old state, the step's rows).
//
// u has `row_in` values per row (the convolved channels are its first C), y is dense [N, C]; w float32 [taps, C] (tap
// by tap, so that neighbouring channels' weights are neighbours).
#include "common.cuh"

namespace {

template <typename T> __device__ __forceinline__ float finish(float acc, const float* __restrict__ bias, int c, int silu) {
    if (bias != nullptr) acc += bias[c];
    return silu ? silu_for<T>(acc) : acc;
}

// VEC channels a thread (16 bytes of a row where the sizes allow it, else one).
template <typename T, int VEC>
__global__ void short_conv_kernel(const T* __restrict__ u, int64_t row_in, const float* __restrict__ w, const float* __restrict__ state,
                                  int64_t slot_stride, const int* __restrict__ token_seq, const int* __restrict__ seq_start,
                                  const int* __restrict__ seq_slots, T* __restrict__ y, int C, int taps, int64_t n_tokens,
                                  const float* __restrict__ bias, int silu) {
    pdl_launch_dependents();
    pdl_wait();
    const int per_row = C / VEC;
    const int64_t total = n_tokens * per_row;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t t = i / per_row;
        const int c = (int)(i % per_row) * VEC;
        const int seq = token_seq[t];
        const int64_t first = seq_start[seq];                  // the step's first row of this sequence
        const float* st = state + (int64_t)seq_slots[seq] * slot_stride;
        float acc[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) acc[k] = 0.0f;
        for (int j = 0; j < taps; ++j) {
            const int64_t src = t - (taps - 1) + j;
            float x[VEC];
            if (src >= first) {
                if constexpr (VEC == 1) {
                    x[0] = to_f32<T>(u[src * row_in + c]);
                } else {
                    const Pack<T> pk = load_pack<T>(u + src * row_in + c);
#pragma unroll
                    for (int k = 0; k < VEC; ++k) x[k] = pk.get(k);
                }
            } else {
#pragma unroll
                for (int k = 0; k < VEC; ++k) x[k] = st[(int64_t)(taps - 1 + (src - first)) * C + c + k];
            }
#pragma unroll
            for (int k = 0; k < VEC; ++k) acc[k] = fmaf(w[(int64_t)j * C + c + k], x[k], acc[k]);
        }
        if constexpr (VEC == 1) {
            y[t * C + c] = from_f32<T>(finish<T>(acc[0], bias, c, silu));
        } else {
            Pack<T> pk;
#pragma unroll
            for (int k = 0; k < VEC; ++k) pk.set(k, finish<T>(acc[k], bias, c + k, silu));
            store_pack<T>(y + t * C + c, pk);
        }
    }
}

// The same for TAPS known at compile time and 16-byte packets: a thread walks `run` consecutive tokens of its VEC channels
// with the last TAPS - 1 rows in registers, so that every row is read once (and TAPS - 1 more at the start of a run or of a
// sequence).  The sums run in the same order as above: the same bits.
template <typename T, int VEC, int TAPS>
__global__ void short_conv_walk_kernel(const T* __restrict__ u, int64_t row_in, const float* __restrict__ w, const float* __restrict__ state,
                                       int64_t slot_stride, const int* __restrict__ token_seq, const int* __restrict__ seq_start,
                                       const int* __restrict__ seq_slots, T* __restrict__ y, int C, int64_t n_tokens, int run,
                                       const float* __restrict__ bias, int silu) {
    pdl_launch_dependents();
    pdl_wait();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (c >= C) return;
    float wt[TAPS][VEC], win[TAPS > 1 ? TAPS - 1 : 1][VEC], add[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) add[k] = bias != nullptr ? bias[c + k] : 0.0f;
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
        for (int k = 0; k < VEC; ++k) wt[j][k] = w[(int64_t)j * C + c + k];
    const int64_t t_begin = (int64_t)blockIdx.y * run, t_end = min(t_begin + run, n_tokens);
    auto fill = [&](int64_t t, int seq) {                      // the rows before token t
        const int64_t first = seq_start[seq];
        const float* st = state + (int64_t)seq_slots[seq] * slot_stride;
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) {
            const int64_t src = t - (TAPS - 1) + j;
            if (src >= first) {
                const Pack<T> pk = load_pack<T>(u + src * row_in + c);
#pragma unroll
                for (int k = 0; k < VEC; ++k) win[j][k] = pk.get(k);
            } else {
#pragma unroll
                for (int k = 0; k < VEC; ++k) win[j][k] = st[(int64_t)(TAPS - 1 + (src - first)) * C + c + k];
            }
        }
    };
    auto one = [&](int64_t t, const Pack<T>& pk) {
        float x[VEC], acc[VEC];
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            x[k] = pk.get(k);
            acc[k] = 0.0f;
        }
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
            for (int k = 0; k < VEC; ++k) acc[k] = fmaf(wt[j][k], win[j][k], acc[k]);
        Pack<T> out;
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            acc[k] = fmaf(wt[TAPS - 1][k], x[k], acc[k]);
            acc[k] += add[k];
            if (silu) acc[k] = silu_for<T>(acc[k]);
            out.set(k, acc[k]);
        }
        store_pack<T>(y + t * C + c, out);
#pragma unroll
        for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
            for (int k = 0; k < VEC; ++k) win[j][k] = win[j + 1][k];
        if (TAPS > 1) {
#pragma unroll
            for (int k = 0; k < VEC; ++k) win[TAPS - 2 > 0 ? TAPS - 2 : 0][k] = x[k];
        }
    };
    const int seq0 = token_seq[t_begin];
    if (seq0 == token_seq[t_end - 1]) {                        // one sequence: the rows of several tokens are on their way together
        constexpr int BATCH = 8;
        fill(t_begin, seq0);
        for (int64_t t0 = t_begin; t0 < t_end; t0 += BATCH) {
            Pack<T> pk[BATCH];
#pragma unroll
            for (int n = 0; n < BATCH; ++n)
                if (t0 + n < t_end) pk[n] = load_pack<T>(u + (t0 + n) * row_in + c);
#pragma unroll
            for (int n = 0; n < BATCH; ++n)
                if (t0 + n < t_end) one(t0 + n, pk[n]);
        }
        return;
    }
    int cur = -1;
    for (int64_t t = t_begin; t < t_end; ++t) {
        const int seq = token_seq[t];
        if (seq != cur) {                                      // the run's first token, or a sequence's first: fill the window
            cur = seq;
            fill(t, seq);
        }
        one(t, load_pack<T>(u + t * row_in + c));
    }
}

template <typename T, int VEC>
__global__ void short_conv_step_kernel(const T* __restrict__ u, int64_t row_in, const float* __restrict__ w, float* __restrict__ state,
                                       int64_t slot_stride, const int* __restrict__ seq_start, const int* __restrict__ seq_slots,
                                       T* __restrict__ y, int C, int taps, int n_seqs, const float* __restrict__ bias, int silu) {
    pdl_launch_dependents();
    pdl_wait();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC, seq = blockIdx.y;
    if (c >= C) return;
    const int64_t t = seq_start[seq];
    float* st = state + (int64_t)seq_slots[seq] * slot_stride + c;
    float x[VEC], acc[VEC];
    if constexpr (VEC == 1) {
        x[0] = to_f32<T>(u[t * row_in + c]);
    } else {
        const Pack<T> pk = load_pack<T>(u + t * row_in + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) x[k] = pk.get(k);
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) acc[k] = 0.0f;
    for (int j = 0; j < taps - 1; ++j) {
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            const float old = st[(int64_t)j * C + k];
            acc[k] = fmaf(w[(int64_t)j * C + c + k], old, acc[k]);
            if (j > 0) st[(int64_t)(j - 1) * C + k] = old;
        }
    }
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
        if (taps > 1) st[(int64_t)(taps - 2) * C + k] = x[k];
        acc[k] = finish<T>(fmaf(w[(int64_t)(taps - 1) * C + c + k], x[k], acc[k]), bias, c + k, silu);
    }
    if constexpr (VEC == 1) {
        y[t * C + c] = from_f32<T>(acc[0]);
    } else {
        Pack<T> pk;
#pragma unroll
        for (int k = 0; k < VEC; ++k) pk.set(k, acc[k]);
        store_pack<T>(y + t * C + c, pk);
    }
}

template <typename T, int TAPS>
int short_conv_walk_launch(const T* u, int64_t row_in, const float* w, const float* state, int64_t slot_stride, const int* token_seq,
                           const int* seq_start, const int* seq_slots, T* y, int C, int64_t n_tokens, const float* bias, int silu,
                           cudaStream_t stream) {
    constexpr int V = Pack<T>::N;
    const int run = n_tokens >= 1024 ? 16 : (n_tokens >= 128 ? 4 : 1);
    const int64_t runs = (n_tokens + run - 1) / run;
    if (runs > 65535) return Q3_ERR_TOO_LARGE;
    const dim3 grid((unsigned)((C / V + 127) / 128), (unsigned)runs);
    return (int)q3_launch(short_conv_walk_kernel<T, V, TAPS>, grid, dim3(128), 0, stream, u, row_in, w, state, slot_stride, token_seq,
                          seq_start, seq_slots, y, C, n_tokens, run, bias, silu);
}

template <typename T>
__global__ void short_conv_state_kernel(const T* __restrict__ u, int64_t row_in, float* __restrict__ state, int64_t slot_stride,
                                        const int* __restrict__ seq_start, const int* __restrict__ seq_slots, int C, int taps,
                                        int n_seqs) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t total = (int64_t)n_seqs * C;
    const int keep = taps - 1;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int seq = (int)(i / C), c = (int)(i % C);
        const int64_t first = seq_start[seq], n_new = seq_start[seq + 1] - first;
        float* st = state + (int64_t)seq_slots[seq] * slot_stride;
        // row r of the new state is row r + n_new of (old state, new rows): ascending r never reads what it wrote
        for (int r = 0; r < keep; ++r) {
            const int64_t src = r + n_new;
            st[(int64_t)r * C + c] = src < keep ? st[src * C + c] : to_f32<T>(u[(first + src - keep) * row_in + c]);
        }
    }
}

template <typename T>
int short_conv_launch(const T* u, int64_t row_in, const float* w, float* state, int64_t slot_stride, const int* token_seq, const int* seq_start,
                      const int* seq_slots, T* y, int C, int taps, int64_t n_tokens, int n_seqs, const float* bias, int silu,
                      int single, cudaStream_t stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (C <= 0 || taps <= 0 || taps > 64 || row_in < C) return Q3_ERR_BAD_SIZE;
    constexpr int V = Pack<T>::N;
    const bool vec = C % V == 0 && row_in % V == 0 && aligned16(u) && aligned16(y);
    if (single) {
        if (n_tokens != n_seqs || n_seqs > 65535) return Q3_ERR_BAD_SIZE;
        const int packets = C / (vec ? V : 1);
        return (int)q3_launch(vec ? short_conv_step_kernel<T, V> : short_conv_step_kernel<T, 1>, dim3((packets + 63) / 64, n_seqs), dim3(64), 0,
                              stream, u, row_in, w, state, slot_stride, seq_start, seq_slots, y, C, taps, n_seqs, bias, silu);
    }
    int code;
    if (vec && taps >= 2 && taps <= 4 && (n_tokens + 15) / 16 <= 65535) {
        auto walk = [&](auto launch) {
            return launch(u, row_in, w, state, slot_stride, token_seq, seq_start, seq_slots, y, C, n_tokens, bias, silu, stream);
        };
        code = taps == 2 ? walk(short_conv_walk_launch<T, 2>) : (taps == 3 ? walk(short_conv_walk_launch<T, 3>) : walk(short_conv_walk_launch<T, 4>));
    } else {
        const int64_t blocks = (n_tokens * (C / (vec ? V : 1)) + 255) / 256;
        code = (int)q3_launch(vec ? short_conv_kernel<T, V> : short_conv_kernel<T, 1>, dim3((unsigned)(blocks < 65536 ? blocks : 65536)),
                              dim3(256), 0, stream, u, row_in, w, (const float*)state, slot_stride, token_seq, seq_start, seq_slots, y, C,
                              taps, n_tokens, bias, silu);
    }
    if (code != 0 || taps == 1) return code;
    const int64_t blocks = ((int64_t)n_seqs * C + 255) / 256;
    return (int)q3_launch(short_conv_state_kernel<T>, dim3((unsigned)(blocks < 65536 ? blocks : 65536)), dim3(256), 0, stream, u, row_in,
                          state, slot_stride, seq_start, seq_slots, C, taps, n_seqs);
}

}  // namespace

#define Q3_CONV_EXPORTS(SUFFIX, T)                                                                                        \
    Q3_EXPORT int q3_short_conv_##SUFFIX(const void* u, int64_t row_in, const float* w, float* state, int64_t slot_stride, \
                                         const int* token_seq, const int* seq_start, const int* seq_slots, void* y,      \
                                         int channels, int taps, int64_t n_tokens, int n_seqs, const float* bias,        \
                                         int silu, int single, void* stream) {                                            \
        return short_conv_launch<T>((const T*)u, row_in, w, state, slot_stride, token_seq, seq_start, seq_slots, (T*)y,   \
                                    channels, taps, n_tokens, n_seqs, bias, silu, single, (cudaStream_t)stream);          \
    }

Q3_CONV_EXPORTS(f32, float)
Q3_CONV_EXPORTS(bf16, bf16)

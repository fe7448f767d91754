// Attention over the paged cache, in its general form: any head size in steps of 16 up
// to 256, any number of heads and groups, any mix of prompt and decode tokens in one
// launch, float or bf16 elements with 32-bit scores, softmax and sums.  It is the
// 32-bit path's attention and the fallback of the bf16 path for head sizes that the
// tensor-core kernels do not take.
//
//   qkv_prepare : per-head RMSNorm of q and k, rotation, and the write of k and v
//                 into their cache pages - one pass over the projection output where
//                 the reference runs rms_norm x2 (src/model/self_attention.cpp:147-149),
//                 apply_rope x2 (:152, src/ops/rope.cu:60-84) and two strided copies
//                 (src/model/kv_cache.cpp:165-188).
//   attention   : causal grouped-query attention by loop bound, scale after the dot,
//                 online softmax (src/ops/gqa_attention.cu:42-44,84-86,117,119-144,152).
//
// Beyond what Qwen3 needs, as parameters: a bias added to the projection output before the
// rotation; values of another size than keys (`vd`); scores capped smoothly,
// s <- cap * tanh(s / cap); a window of the last keys, or the keys of the query's own chunk
// of positions (chunks of `chunk` positions counted from 0); and a sink, one more term
// exp(0) in the softmax's denominator that carries no value.  Further: values that are the projected keys (no value
// columns in the projection), values rotated by their own position (the caller turns the outputs back), and pooled
// blocks beside a window: every block of `size` tokens that lies wholly before a query's window is seen as one key and
// one value, the means of the block's cached keys and values, which `pool_blocks` makes when a block is complete.
//
// Further still: queries multiplied by a temperature of their position, 1 + coef ln(floor((p + 1) / every) + 1), after
// their norm; and a bias added to every scaled score by the distance between query and key, one number per head and
// distance up to a last one that stands for all that are further.
//
// Cache layout: pages [page, kv head, PAGE tokens, head_dim]; `page_table[seq]` lists
// the pages of a sequence in order.  Keys are visited page by page in ascending
// position, so the result for one (position, head) does not depend on how the tokens
// were cut into steps or on what else is in the batch.
#include "common.cuh"

namespace {

constexpr int PAGE = Q3_PAGE_TOKENS;
constexpr int MAX_HEAD_DIM = 256;
constexpr int GENERIC_KEY_DIM = 1024, GENERIC_VALUE_DIM = 512;   // what the general attention kernel takes

template <typename T> __device__ __forceinline__ void load_pack_f32(const T* p, float (&v)[Pack<T>::N]) {
    const Pack<T> k = load_pack<T>(p);
#pragma unroll
    for (int i = 0; i < Pack<T>::N; ++i) v[i] = k.get(i);
}
template <typename T> __device__ __forceinline__ void store_pack_f32(T* p, const float (&v)[Pack<T>::N]) {
    Pack<T> k;
#pragma unroll
    for (int i = 0; i < Pack<T>::N; ++i) k.set(i, v[i]);
    store_pack<T>(p, k);
}

template <typename T> __device__ __forceinline__ float normed(float unit, float w, int once) {
    return once ? unit * w : round_to<T>(round_to<T>(unit) * w);
}

struct PrepareOptions {
    int64_t row;            // values from one row of the projection to the next
    int tied;               // the values are the projected keys: the projection has no value columns
    int norm_once;          // a normed value is rounded once, when it is stored (else after the division and the weight too)
    const float* v_cos;     // [positions, vd / 2] or null: values are rotated by their position, over the whole head
    const float* v_sin;
    float temp_coef;        // queries are multiplied by 1 + temp_coef ln((pos + 1) / temp_every + 1), a whole quotient (0: by nothing)
    int temp_every;
};

__device__ __forceinline__ float query_temperature(const PrepareOptions& opt, int pos) {
    return 1.0f + opt.temp_coef * logf((float)((pos + 1) / opt.temp_every + 1));
}

// Biases by distance: table [query heads][count], the last column for every distance from count - 1 on (null: none).
struct DistanceBias {
    const float* table;
    int count;
};

template <typename T>
__global__ void qkv_prepare_kernel(const T* __restrict__ qkv, T* __restrict__ q_out, T* __restrict__ k_pages,
                                   T* __restrict__ v_pages, const float* __restrict__ q_norm_w,
                                   const float* __restrict__ k_norm_w, const float* __restrict__ cos_tab,
                                   const float* __restrict__ sin_tab, const int* __restrict__ token_seq,
                                   const int* __restrict__ token_pos, const int* __restrict__ page_table,
                                   int pages_per_seq, int nq, int nkv, int d, float eps, int write_kv, int rot,
                                   const float* __restrict__ bias, int vd, int nv, const PrepareOptions opt) {
    pdl_launch_dependents();
    pdl_wait();
    const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.x * warps + warp;
    if (head >= nq + nkv + nv || (head >= nq && !write_kv)) return;   // a layer that reads another layer's cache writes none
    const int64_t t = blockIdx.y;
    const int pos = token_pos[t];
    // a row of the projection: nq query heads and nkv key heads of d values, then nv value heads of vd values
    int64_t col0 = head < nq + nkv ? (int64_t)head * d : (int64_t)(nq + nkv) * d + (int64_t)(head - nq - nkv) * vd;
    if (opt.tied && head >= nq + nkv) col0 = (int64_t)(head - nkv) * d;
    const T* src = qkv + t * opt.row + col0;
    if (bias != nullptr) bias += col0;

    T* dst;
    const float* norm_w = nullptr;
    bool rotate = cos_tab != nullptr;
    if (head < nq) {
        dst = q_out + t * (int64_t)nq * d + (int64_t)head * d;
        norm_w = q_norm_w;
    } else {
        const bool is_v = head >= nq + nkv;
        const int kvh = is_v ? head - nq - nkv : head - nq;
        const int page = page_table[(int64_t)token_seq[t] * pages_per_seq + pos / PAGE];
        dst = (is_v ? v_pages : k_pages) + (((int64_t)page * (is_v ? nv : nkv) + kvh) * PAGE + pos % PAGE) * (is_v ? vd : d);
        norm_w = is_v ? nullptr : k_norm_w;
        rotate = rotate && !is_v;
        if (is_v) {                                     // a value head: vd values that pass through
            d = vd;
            cos_tab = opt.v_cos;
            sin_tab = opt.v_sin;
            rotate = cos_tab != nullptr;
            rot = rotate ? vd : 0;
        }
    }

    // The first `rot` values of the head are rotated in pairs (i, i + rot/2), i = lane + 32 n; the values from
    // `rot` on (none when the whole head is rotated, as in Qwen3) are normalised and pass through.
    const int rhalf = rot >> 1;
    float a[MAX_HEAD_DIM / 64], b[MAX_HEAD_DIM / 64], c[MAX_HEAD_DIM / 32];
    float sq = 0.0f;
#pragma unroll
    for (int n = 0; n < MAX_HEAD_DIM / 64; ++n) {
        const int i = lane + 32 * n;
        a[n] = b[n] = 0.0f;
        if (i < rhalf) {
            a[n] = to_f32<T>(src[i]);
            b[n] = to_f32<T>(src[i + rhalf]);
            if (bias != nullptr) {
                a[n] = round_to<T>(a[n] + bias[i]);
                b[n] = round_to<T>(b[n] + bias[i + rhalf]);
            }
            sq += a[n] * a[n] + b[n] * b[n];
        }
    }
    if (rot < d) {
#pragma unroll
        for (int n = 0; n < MAX_HEAD_DIM / 32; ++n) {
            const int i = rot + lane + 32 * n;
            c[n] = 0.0f;
            if (i < d) {
                c[n] = to_f32<T>(src[i]);
                if (bias != nullptr) c[n] = round_to<T>(c[n] + bias[i]);
                sq += c[n] * c[n];
            }
        }
    }
    if (norm_w != nullptr) {
        const float inv = rsqrtf(warp_sum(sq) / (float)d + eps);
#pragma unroll
        for (int n = 0; n < MAX_HEAD_DIM / 64; ++n) {
            const int i = lane + 32 * n;
            if (i < rhalf) {
                a[n] = normed<T>(a[n] * inv, norm_w[i], opt.norm_once);
                b[n] = normed<T>(b[n] * inv, norm_w[i + rhalf], opt.norm_once);
            }
        }
        if (rot < d) {
#pragma unroll
            for (int n = 0; n < MAX_HEAD_DIM / 32; ++n) {
                const int i = rot + lane + 32 * n;
                if (i < d) c[n] = normed<T>(c[n] * inv, norm_w[i], opt.norm_once);
            }
        }
    }
    if (opt.temp_coef != 0.0f && head < nq) {
        const float temp = query_temperature(opt, pos);
#pragma unroll
        for (int n = 0; n < MAX_HEAD_DIM / 64; ++n) {
            a[n] *= temp;
            b[n] *= temp;
        }
        if (rot < d) {
#pragma unroll
            for (int n = 0; n < MAX_HEAD_DIM / 32; ++n) c[n] *= temp;
        }
    }
#pragma unroll
    for (int n = 0; n < MAX_HEAD_DIM / 64; ++n) {
        const int i = lane + 32 * n;
        if (i < rhalf) {
            float x = a[n], y = b[n];
            if (rotate) {
                const float cs = cos_tab[(int64_t)pos * rhalf + i], sn = sin_tab[(int64_t)pos * rhalf + i];
                x = a[n] * cs - b[n] * sn;
                y = b[n] * cs + a[n] * sn;
            }
            dst[i] = from_f32<T>(x);
            dst[i + rhalf] = from_f32<T>(y);
        }
    }
    if (rot < d) {
#pragma unroll
        for (int n = 0; n < MAX_HEAD_DIM / 32; ++n) {
            const int i = rot + lane + 32 * n;
            if (i < d) dst[i] = from_f32<T>(c[n]);
        }
    }
}

// The same with 16-byte accesses: a head is shared by (d/2)/VEC lanes.  The lanes of the rotated stretch own VEC
// consecutive elements of its first half and the matching VEC of its second half (the two members of every rotation
// pair), the lanes behind them 2 VEC consecutive elements that pass through; a warp works on several heads at once.
// One warp per group of consecutive (token, head) pairs.
template <typename T>
__global__ void qkv_prepare_vec_kernel(const T* __restrict__ qkv, T* __restrict__ q_out, T* __restrict__ k_pages,
                                       T* __restrict__ v_pages, const float* __restrict__ q_norm_w,
                                       const float* __restrict__ k_norm_w, const float* __restrict__ cos_tab,
                                       const float* __restrict__ sin_tab, const int* __restrict__ token_seq,
                                       const int* __restrict__ token_pos, const int* __restrict__ page_table,
                                       int pages_per_seq, int nq, int nkv, int d, float eps, int write_kv, int rot,
                                       int64_t n_tokens, const float* __restrict__ bias, const PrepareOptions opt) {
    constexpr int VEC = Pack<T>::N;
    pdl_launch_dependents();
    pdl_wait();
    const int lph = (d >> 1) / VEC, hpw = 32 / lph;                   // lanes per head, heads per warp
    const int lane = threadIdx.x & 31, sub = lane % lph, grp = lane / lph;
    const int heads = write_kv ? nq + 2 * nkv : nq;
    const int64_t warp = (int64_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int64_t pair = warp * hpw + grp;                             // flat (token, head) index
    const bool active = grp < hpw && pair < n_tokens * heads;
    const int64_t t = active ? pair / heads : 0;
    const int head = active ? (int)(pair % heads) : 0;
    const bool is_q = head < nq, is_v = head >= nq + nkv;
    const bool live = active && (is_q || write_kv);
    const int pos = token_pos[t];
    const float* cs_tab = is_v ? opt.v_cos : cos_tab;
    const float* sn_tab = is_v ? opt.v_sin : sin_tab;
    const int rhalf = (is_v ? d : rot) >> 1, turning = rhalf / VEC;    // a value head is rotated as a whole, or not at all
    const bool rotate = cs_tab != nullptr && sub < turning;
    const int a_at = sub < turning ? sub * VEC : 2 * rhalf + (sub - turning) * 2 * VEC;
    const int b_at = sub < turning ? rhalf + sub * VEC : a_at + VEC;
    const int col = (opt.tied && is_v ? head - nkv : head) * d;        // the head's columns in a row of the projection
    const T* src = qkv + t * opt.row + col;
    float a[VEC], b[VEC];
#pragma unroll
    for (int i = 0; i < VEC; ++i) a[i] = b[i] = 0.0f;
    if (live) {
        load_pack_f32<T>(src + a_at, a);
        load_pack_f32<T>(src + b_at, b);
        if (bias != nullptr) {                       // one value per column of the projection, added before anything else
            const float* bh = bias + col;
#pragma unroll
            for (int i = 0; i < VEC; ++i) {
                a[i] = round_to<T>(a[i] + bh[a_at + i]);
                b[i] = round_to<T>(b[i] + bh[b_at + i]);
            }
        }
    }
    const float* norm_w = is_q ? q_norm_w : (is_v ? nullptr : k_norm_w);
    // the sum over the lanes of a head: every lane of the warp takes part in every shuffle
    float sq = 0.0f;
#pragma unroll
    for (int i = 0; i < VEC; ++i) sq += a[i] * a[i] + b[i] * b[i];
    float total = 0.0f;
    const int first = grp * lph;
    for (int j = 0; j < lph; ++j) total += __shfl_sync(0xffffffffu, sq, (first + j) & 31);
    if (norm_w != nullptr) {
        const float inv = rsqrtf(total / (float)d + eps);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            a[i] = normed<T>(a[i] * inv, norm_w[a_at + i], opt.norm_once);
            b[i] = normed<T>(b[i] * inv, norm_w[b_at + i], opt.norm_once);
        }
    }
    if (!live) return;
    if (opt.temp_coef != 0.0f && is_q) {
        const float temp = query_temperature(opt, pos);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            a[i] *= temp;
            b[i] *= temp;
        }
    }
    if (rotate) {
        const float* c = cs_tab + (int64_t)pos * rhalf + a_at;
        const float* sn = sn_tab + (int64_t)pos * rhalf + a_at;
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
            const float x = a[i] * c[i] - b[i] * sn[i], y = b[i] * c[i] + a[i] * sn[i];
            a[i] = x;
            b[i] = y;
        }
    }
    T* dst;
    if (is_q) {
        dst = q_out + (t * nq + head) * (int64_t)d;
    } else {
        const int kvh = (head - nq) % nkv;
        const int page = page_table[(int64_t)token_seq[t] * pages_per_seq + pos / PAGE];
        dst = (is_v ? v_pages : k_pages) + (((int64_t)page * nkv + kvh) * PAGE + pos % PAGE) * d;
    }
    store_pack_f32<T>(dst + a_at, a);
    store_pack_f32<T>(dst + b_at, b);
}

// The pooled blocks that the step completes: block b of a sequence holds the tokens b size .. b size + size - 1, all of
// them in the cache by now; its key and value are the means of theirs, and go to entry b of the sequence's pool pages.
// One block of threads per (block of tokens, key/value head, sequence); thread i owns one key or value channel.
template <typename T>
__global__ void pool_blocks_kernel(const T* __restrict__ k_pages, const T* __restrict__ v_pages, const int* __restrict__ page_table,
                                   T* __restrict__ pool_k, T* __restrict__ pool_v, const int* __restrict__ pool_table,
                                   const int* __restrict__ seq_start, const int* __restrict__ seq_pos0, int pages_per_seq, int nkv,
                                   int d, int vd, int size) {
    pdl_launch_dependents();
    pdl_wait();
    const int kvh = blockIdx.y, seq = blockIdx.z;
    const int64_t pos0 = seq_pos0[seq], end = pos0 + seq_start[seq + 1] - seq_start[seq];
    const int64_t b = pos0 / size + blockIdx.x;
    if ((b + 1) * size > end) return;
    const int* pages = page_table + (int64_t)seq * pages_per_seq;
    const int64_t to = ((int64_t)pool_table[(int64_t)seq * pages_per_seq + b / PAGE] * nkv + kvh) * PAGE + b % PAGE;
    const float inv = 1.0f / (float)size;
    for (int i = threadIdx.x; i < d + vd; i += blockDim.x) {
        const bool is_v = i >= d;
        const int c = is_v ? i - d : i, width = is_v ? vd : d;
        const T* from = (is_v ? v_pages : k_pages) + c;
        float sum = 0.0f;
#pragma unroll 4
        for (int j = 0; j < size; ++j) {
            const int64_t p = b * size + j;
            sum += to_f32<T>(from[(((int64_t)pages[p / PAGE] * nkv + kvh) * PAGE + p % PAGE) * width]);
        }
        (is_v ? pool_v : pool_k)[to * width + c] = from_f32<T>(sum * inv);
    }
}

// Pooled blocks beside a window (size 0: none): entry b of a sequence's pool pages is seen by a query whose window
// starts at `lo` if the block's last token lies before it, that is if b < lo / size.
template <typename T> struct PoolView {
    const T* k;
    const T* v;
    const int* table;           // [sequences, pages_per_seq]
    int size;
};

// One block per (query head, token).  128 threads: the four warps share the keys of a
// page for the scores; thread t owns output dims t, t + 128, t + 256 and t + 384.  Keys up to GENERIC_KEY_DIM and
// values up to GENERIC_VALUE_DIM wide: the rows of a latent cache (one wide key/value head for all query heads).
template <typename T>
__global__ void __launch_bounds__(128)
attention_generic_kernel(const T* __restrict__ q, const T* __restrict__ k_pages, const T* __restrict__ v_pages,
                         T* __restrict__ out, const int* __restrict__ token_seq, const int* __restrict__ token_pos,
                         const int* __restrict__ page_table, int pages_per_seq, int nq, int nkv, int d, float scale,
                         int window, int vd, float softcap, int chunk, int sink, int nv, int out_f32,
                         const float* __restrict__ sink_values, int keep_first, const PoolView<T> pool, const DistanceBias bias) {
    __shared__ float q_s[GENERIC_KEY_DIM];
    __shared__ float score[PAGE];
    __shared__ float prob[PAGE];
    pdl_launch_dependents();
    pdl_wait();
    const int head = blockIdx.x, kvh = head / (nq / nkv), vh = kvh / (nkv / nv);   // nv value heads: each serves nkv / nv key heads
    const int64_t t = blockIdx.y;
    const int pos = token_pos[t];
    const int* pages = page_table + (int64_t)token_seq[t] * pages_per_seq;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

    for (int i = tid; i < d; i += 128) q_s[i] = to_f32<T>(q[(t * nq + head) * (int64_t)d + i]);
    __syncthreads();

    const int lo = window > 0 ? max(0, pos - window + 1) : (chunk > 0 ? pos / chunk * chunk : 0);
    // the sink is a key without a value whose score is 0, or the head's own number (`sink_values`), neither scaled
    // nor capped: the running maximum and sum start from it
    float m_run = sink ? (sink_values ? sink_values[head] : 0.0f) : -INFINITY, l_run = sink ? 1.0f : 0.0f;
    float acc[GENERIC_VALUE_DIM / 128] = {};
    const float inv_cap = softcap > 0.0f ? 1.0f / softcap : 0.0f;
    // with a window, the first `keep_first` keys of the sequence stay visible: their pages come first, then the window's
    const int keep = window > 0 ? keep_first : 0;
    // the pooled blocks' pages come first of all
    const int n_blocks = pool.size > 0 ? lo / pool.size : 0, pool_pages = (n_blocks + PAGE - 1) / PAGE;
    const int* pool_list = pool.size > 0 ? pool.table + (int64_t)token_seq[t] * pages_per_seq : nullptr;
    for (int x = 0; x <= pool_pages + pos / PAGE; ++x) {
        const bool pooled = x < pool_pages;
        const int pg = pooled ? x : x - pool_pages;
        if (!pooled && pg < lo / PAGE && pg * PAGE >= keep) continue;   // nothing of this page is seen (it may be given back)
        const int page = pooled ? pool_list[pg] : pages[pg];
        const T* kp = (pooled ? pool.k : k_pages) + ((int64_t)page * nkv + kvh) * PAGE * d;
        const T* vp = (pooled ? pool.v : v_pages) + ((int64_t)page * nv + vh) * PAGE * vd;
        const int j_hi = min((pooled ? n_blocks - 1 : pos) - pg * PAGE, PAGE - 1);            // inclusive, in-page
        const int j_lo = pooled || pg * PAGE < keep ? 0 : max(lo - pg * PAGE, 0);
        const int gap_lo = pooled ? PAGE : keep - pg * PAGE;            // keys j with gap_lo <= j < gap_hi are not seen
        const int gap_hi = pooled ? PAGE : lo - pg * PAGE;
        for (int j = warp; j < PAGE; j += 4) {
            float dot = 0.0f;
            if (j >= j_lo && j <= j_hi && !(j >= gap_lo && j < gap_hi)) {
                for (int i = lane; i < d; i += 32) dot = fmaf(q_s[i], to_f32<T>(kp[(int64_t)j * d + i]), dot);
            }
            dot = warp_sum(dot) * scale;
            if (softcap > 0.0f) dot = softcap * tanhf(dot * inv_cap);
            if (bias.table != nullptr) dot += bias.table[(int64_t)head * bias.count + min(max(pos - pg * PAGE - j, 0), bias.count - 1)];
            if (lane == 0) score[j] = (j >= j_lo && j <= j_hi && !(j >= gap_lo && j < gap_hi)) ? dot : -INFINITY;
        }
        __syncthreads();
        float m_new = m_run;
        for (int j = 0; j < PAGE; ++j) m_new = fmaxf(m_new, score[j]);
        if (tid < PAGE) prob[tid] = score[tid] > -INFINITY ? expf(score[tid] - m_new) : 0.0f;
        __syncthreads();
        const float alpha = expf(m_run - m_new);  // 0 on the first page (m_run = -inf, m_new finite)
        float l_add = 0.0f, v_add[GENERIC_VALUE_DIM / 128] = {};
        for (int j = j_lo; j <= j_hi; ++j) {
            const float p = prob[j];
            l_add += p;
#pragma unroll
            for (int n = 0; n < GENERIC_VALUE_DIM / 128; ++n)
                if (tid + n * 128 < vd) v_add[n] = fmaf(p, to_f32<T>(vp[(int64_t)j * vd + tid + n * 128]), v_add[n]);
        }
        l_run = l_run * alpha + l_add;
#pragma unroll
        for (int n = 0; n < GENERIC_VALUE_DIM / 128; ++n) acc[n] = acc[n] * alpha + v_add[n];
        m_run = m_new;
        __syncthreads();  // score/prob are rewritten by the next page
    }
    if (out_f32) {                                   // the caller goes on in 32-bit (differences of attention maps)
        float* o = reinterpret_cast<float*>(out) + (t * nq + head) * (int64_t)vd;
#pragma unroll
        for (int n = 0; n < GENERIC_VALUE_DIM / 128; ++n)
            if (tid + n * 128 < vd) o[tid + n * 128] = acc[n] / l_run;
        return;
    }
    T* o = out + (t * nq + head) * (int64_t)vd;
#pragma unroll
    for (int n = 0; n < GENERIC_VALUE_DIM / 128; ++n)
        if (tid + n * 128 < vd) o[tid + n * 128] = from_f32<T>(acc[n] / l_run);
}

template <typename T>
int qkv_prepare_launch(const T* qkv, T* q_out, T* k_pages, T* v_pages, const float* q_norm_w, const float* k_norm_w,
                       const float* cos_tab, const float* sin_tab, const int* token_seq, const int* token_pos,
                       const int* page_table, int pages_per_seq, int64_t n_tokens, int nq, int nkv, int d, float eps,
                       int write_kv, int rot, const float* bias, int vd, int nv, PrepareOptions opt, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (nv <= 0) nv = nkv;                       // as many value heads as key heads
    if (d <= 0 || d > MAX_HEAD_DIM || nq <= 0 || nkv <= 0 || nkv % nv != 0) return Q3_ERR_BAD_SIZE;
    if (rot <= 0) rot = d;                       // the whole head is rotated
    if (rot > d || (rot % 2 != 0 && (cos_tab != nullptr || rot != d))) return Q3_ERR_BAD_SIZE;   // pairs need an even count
    if (rot % 2 != 0) rot = 0;                   // an odd head without tables: every value passes through
    if (vd <= 0) vd = d;                         // values as wide as keys
    if (vd > MAX_HEAD_DIM) return Q3_ERR_BAD_SIZE;
    // a projection of the queries alone is enough when no key is written
    const int64_t columns = write_kv ? (int64_t)(nq + nkv) * d + (opt.tied ? 0 : (int64_t)nv * vd) : (int64_t)nq * d;
    if (opt.temp_coef != 0.0f && opt.temp_every <= 0) return Q3_ERR_BAD_SIZE;
    if (opt.row <= 0) opt.row = columns;
    if (opt.row < columns || (opt.tied && (vd != d || nv != nkv)) || (opt.v_cos == nullptr) != (opt.v_sin == nullptr) ||
        (opt.v_cos != nullptr && vd % 2 != 0))
        return Q3_ERR_BAD_SIZE;
    constexpr int VEC = Pack<T>::N;
    if ((rot / 2) % VEC == 0 && (d - rot) % (2 * VEC) == 0 && rot % 2 == 0 && ((vd == d && nv == nkv) || !write_kv) && n_tokens >= 64 && (d / 2) % VEC == 0 &&
        (d / 2) / VEC <= 32 && opt.row % VEC == 0 && aligned16(qkv) && aligned16(q_out) && aligned16(k_pages) && aligned16(v_pages)) {
        const int hpw = 32 / ((d / 2) / VEC);
        const int64_t n_warps = (n_tokens * (write_kv ? nq + 2 * nkv : nq) + hpw - 1) / hpw;
        const int64_t blocks = (n_warps + 7) / 8;
        if (blocks > 0x7fffffffLL) return Q3_ERR_TOO_LARGE;
        return (int)q3_launch(qkv_prepare_vec_kernel<T>, dim3((unsigned)blocks), dim3(256), 0, stream, qkv, q_out, k_pages,
                              v_pages, q_norm_w, k_norm_w, cos_tab, sin_tab, token_seq, token_pos, page_table, pages_per_seq,
                              nq, nkv, d, eps, write_kv, rot, n_tokens, bias, opt);
    }
    if (n_tokens > 65535) return Q3_ERR_TOO_LARGE;
    const int warps = 4;
    const dim3 grid(((write_kv ? nq + nkv + nv : nq) + warps - 1) / warps, (unsigned)n_tokens);
    return (int)q3_launch(qkv_prepare_kernel<T>, grid, dim3(warps * 32), 0, stream, qkv, q_out, k_pages, v_pages, q_norm_w,
                          k_norm_w, cos_tab, sin_tab, token_seq, token_pos, page_table, pages_per_seq, nq, nkv, d, eps, write_kv, rot,
                          bias, vd, nv, opt);
}

template <typename T>
int attention_generic_launch(const T* q, const T* k_pages, const T* v_pages, T* out, const int* token_seq,
                             const int* token_pos, const int* page_table, int pages_per_seq, int64_t n_tokens, int nq,
                             int nkv, int d, float scale, int window, int vd, float softcap, int chunk, int sink, int nv,
                             int out_f32, const float* sink_values, int keep_first, PoolView<T> pool, DistanceBias bias, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (bias.table != nullptr && (bias.count <= 0 || pool.size > 0)) return Q3_ERR_BAD_SIZE;
    if (pool.size < 0 || (pool.size > 0 && (window <= 0 || keep_first > 0 || pool.k == nullptr || pool.v == nullptr || pool.table == nullptr)))
        return Q3_ERR_BAD_SIZE;
    if (vd <= 0) vd = d;
    if (nv <= 0) nv = nkv;
    if (nkv <= 0 || nkv % nv != 0) return Q3_ERR_BAD_SIZE;
    if (d <= 0 || d > GENERIC_KEY_DIM || vd > GENERIC_VALUE_DIM || nq <= 0 || nkv <= 0 || nq % nkv != 0) return Q3_ERR_BAD_SIZE;
    if ((window > 0 && chunk > 0) || keep_first < 0) return Q3_ERR_BAD_SIZE;
    if (n_tokens > 65535) return Q3_ERR_TOO_LARGE;
    const dim3 grid(nq, (unsigned)n_tokens);
    return (int)q3_launch(attention_generic_kernel<T>, grid, dim3(128), 0, stream, q, k_pages, v_pages, out, token_seq,
                          token_pos, page_table, pages_per_seq, nq, nkv, d, scale, window, vd, softcap, chunk, sink, nv, out_f32, sink_values,
                          keep_first, pool, bias);
}

template <typename T>
int pool_blocks_launch(const T* k_pages, const T* v_pages, const int* page_table, T* pool_k, T* pool_v, const int* pool_table,
                       const int* seq_start, const int* seq_pos0, int pages_per_seq, int n_seqs, int max_new, int nkv, int d, int vd,
                       int size, cudaStream_t stream) {
    if (n_seqs <= 0 || max_new <= 0) return 0;
    if (nkv <= 0 || d <= 0 || vd <= 0 || size <= 0) return Q3_ERR_BAD_SIZE;
    if (n_seqs > 65535 || nkv > 65535) return Q3_ERR_TOO_LARGE;
    // a step of n tokens completes at most n / size blocks, and one more that an earlier step began
    const int threads = d + vd <= 64 ? 64 : (d + vd <= 128 ? 128 : 256);
    return (int)q3_launch(pool_blocks_kernel<T>, dim3((unsigned)(max_new / size + 1), nkv, n_seqs), dim3(threads), 0, stream, k_pages, v_pages,
                          page_table, pool_k, pool_v, pool_table, seq_start, seq_pos0, pages_per_seq, nkv, d, vd, size);
}

// Values blended across layers, on the value columns of a projection's rows (in place): v <- v + bias first (if
// any); the first layer of a chain keeps a copy, `first` [N, width]; a later one goes on with
// v <- (1 - lambda) v + lambda first.  32-bit arithmetic, stored in T.
template <typename T, int VEC>
__global__ void value_mix_kernel(T* __restrict__ rows, int64_t row, int64_t v_off, int width, const float* __restrict__ bias,
                                 T* __restrict__ first, int save, float lambda, int64_t n_tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const int per_row = width / VEC;
    const int64_t total = n_tokens * per_row;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t t = i / per_row;
        const int c = (int)(i % per_row) * VEC;
        T* at = rows + t * row + v_off + c;
        float v[VEC], f[VEC];
        if constexpr (VEC == 1) v[0] = to_f32<T>(*at); else load_pack_f32<T>(at, v);
        if (bias != nullptr) {
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[k] = round_to<T>(v[k] + bias[c + k]);
        }
        if (save) {
            if constexpr (VEC == 1) first[t * width + c] = from_f32<T>(v[0]); else store_pack_f32<T>(first + t * width + c, v);
        } else {
            if constexpr (VEC == 1) f[0] = to_f32<T>(first[t * width + c]); else load_pack_f32<T>(first + t * width + c, f);
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[k] = (1.0f - lambda) * v[k] + lambda * f[k];
        }
        if constexpr (VEC == 1) *at = from_f32<T>(v[0]); else store_pack_f32<T>(at, v);
    }
}

// One sigmoid gate per (token, head) on the attention's output, in place: x[t, h, :] *= sigmoid(gate[t, h]).
template <typename T, int VEC>
__global__ void head_gate_kernel(T* __restrict__ x, const T* __restrict__ gate, int64_t gate_row, int heads, int vd, int64_t n_tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const int per_head = vd / VEC;
    const int64_t total = n_tokens * heads * per_head;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t th = i / per_head, t = th / heads;
        const int h = (int)(th % heads);
        const float z = to_f32<T>(gate[t * gate_row + h]);
        const float g = 1.0f / (1.0f + expf(-z));
        T* at = x + i * VEC;
        float v[VEC];
        if constexpr (VEC == 1) v[0] = to_f32<T>(*at); else load_pack_f32<T>(at, v);
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[k] *= g;
        if constexpr (VEC == 1) *at = from_f32<T>(v[0]); else store_pack_f32<T>(at, v);
    }
}

// The heads of an attention's output, in place: turned back by the query's position (pairs (i, i + vd/2), tables
// [positions, vd/2]; null: not turned) and multiplied value by value by sigmoid(gate) (null: no gate).
template <typename T, int VEC>
__global__ void turn_back_gate_kernel(T* __restrict__ x, const float* __restrict__ cos_tab, const float* __restrict__ sin_tab,
                                      const int* __restrict__ token_pos, const T* __restrict__ gate, int64_t gate_row, int heads, int vd,
                                      int64_t n_tokens) {
    pdl_launch_dependents();
    pdl_wait();
    const int half = vd >> 1, per_head = half / VEC;
    const int64_t total = n_tokens * heads * per_head;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t th = i / per_head, t = th / heads;
        const int c = (int)(i % per_head) * VEC, h = (int)(th % heads);
        T* at = x + th * vd + c;
        float a[VEC], b[VEC];
        if constexpr (VEC == 1) {
            a[0] = to_f32<T>(at[0]);
            b[0] = to_f32<T>(at[half]);
        } else {
            load_pack_f32<T>(at, a);
            load_pack_f32<T>(at + half, b);
        }
        if (cos_tab != nullptr) {
            const float* cs = cos_tab + (int64_t)token_pos[t] * half + c;
            const float* sn = sin_tab + (int64_t)token_pos[t] * half + c;
#pragma unroll
            for (int k = 0; k < VEC; ++k) {
                const float u = a[k] * cs[k] + b[k] * sn[k], v = b[k] * cs[k] - a[k] * sn[k];
                a[k] = u;
                b[k] = v;
            }
        }
        if (gate != nullptr) {
            const T* g = gate + t * gate_row + (int64_t)h * vd + c;
            float ga[VEC], gb[VEC];
            if constexpr (VEC == 1) {
                ga[0] = to_f32<T>(g[0]);
                gb[0] = to_f32<T>(g[half]);
            } else {
                load_pack_f32<T>(g, ga);
                load_pack_f32<T>(g + half, gb);
            }
#pragma unroll
            for (int k = 0; k < VEC; ++k) {
                a[k] *= 1.0f / (1.0f + expf(-ga[k]));
                b[k] *= 1.0f / (1.0f + expf(-gb[k]));
            }
        }
        if constexpr (VEC == 1) {
            at[0] = from_f32<T>(a[0]);
            at[half] = from_f32<T>(b[0]);
        } else {
            store_pack_f32<T>(at, a);
            store_pack_f32<T>(at + half, b);
        }
    }
}

template <typename Kernel, typename... Args>
int launch_flat(Kernel kernel, int64_t work, cudaStream_t stream, Args... args) {
    int64_t blocks = (work + 255) / 256;
    const int64_t resident = (int64_t)q3_device_sm_count() * 16;
    if (blocks > resident) blocks = resident;
    return (int)q3_launch(kernel, dim3((unsigned)blocks), dim3(256), 0, stream, args...);
}

}  // namespace

#define Q3_ATTENTION_EXPORTS(SUFFIX, T)                                                                               \
    Q3_EXPORT int q3_qkv_prepare_##SUFFIX(const void* qkv, void* q_out, void* k_pages, void* v_pages,                  \
                                          const float* q_norm_w, const float* k_norm_w, const float* cos_tab,         \
                                          const float* sin_tab, const int* token_seq, const int* token_pos,           \
                                          const int* page_table, int pages_per_seq, int64_t n_tokens, int nq,         \
                                          int nkv, int d, float eps, int write_kv, int rotary_dim,           \
                                          const float* bias, int value_dim, int value_heads, int64_t row,             \
                                          int tied_values, int norm_once, const float* v_cos, const float* v_sin,     \
                                          float temp_coef, int temp_every, void* stream) {                            \
        PrepareOptions opt;                                                                                           \
        opt.temp_coef = temp_coef; opt.temp_every = temp_every;                                                       \
        opt.row = row; opt.tied = tied_values; opt.norm_once = norm_once; opt.v_cos = v_cos; opt.v_sin = v_sin;       \
        return qkv_prepare_launch<T>((const T*)qkv, (T*)q_out, (T*)k_pages, (T*)v_pages, q_norm_w, k_norm_w, cos_tab, \
                                     sin_tab, token_seq, token_pos, page_table, pages_per_seq, n_tokens, nq, nkv, d,  \
                                     eps, write_kv, rotary_dim, bias, value_dim, value_heads, opt,                    \
                                     (cudaStream_t)stream);                                                           \
    }                                                                                                                 \
    Q3_EXPORT int q3_pool_blocks_##SUFFIX(const void* k_pages, const void* v_pages, const int* page_table, void* pool_k, \
                                          void* pool_v, const int* pool_table, const int* seq_start,                  \
                                          const int* seq_pos0, int pages_per_seq, int n_seqs, int max_new, int nkv,   \
                                          int d, int value_dim, int size, void* stream) {                             \
        return pool_blocks_launch<T>((const T*)k_pages, (const T*)v_pages, page_table, (T*)pool_k, (T*)pool_v,        \
                                     pool_table, seq_start, seq_pos0, pages_per_seq, n_seqs, max_new, nkv, d,         \
                                     value_dim, size, (cudaStream_t)stream);                                          \
    }                                                                                                                 \
    Q3_EXPORT int q3_turn_back_gate_##SUFFIX(void* x, const float* cos_tab, const float* sin_tab, const int* token_pos, \
                                             const void* gate, int64_t gate_row, int heads, int vd, int64_t n_tokens, \
                                             void* stream) {                                                          \
        if (n_tokens <= 0) return 0;                                                                                  \
        if (heads <= 0 || vd <= 0 || vd % 2 != 0 || (cos_tab == nullptr) != (sin_tab == nullptr)) return Q3_ERR_BAD_SIZE; \
        constexpr int V = Pack<T>::N;                                                                                 \
        if ((vd / 2) % V == 0 && aligned16(x) && (gate == nullptr || (gate_row % V == 0 && aligned16(gate))))         \
            return launch_flat(turn_back_gate_kernel<T, V>, n_tokens * heads * (vd / 2 / V), (cudaStream_t)stream,    \
                               (T*)x, cos_tab, sin_tab, token_pos, (const T*)gate, gate_row, heads, vd, n_tokens);    \
        return launch_flat(turn_back_gate_kernel<T, 1>, n_tokens * heads * (vd / 2), (cudaStream_t)stream, (T*)x,     \
                           cos_tab, sin_tab, token_pos, (const T*)gate, gate_row, heads, vd, n_tokens);               \
    }                                                                                                                 \
    Q3_EXPORT int q3_attention_generic_##SUFFIX(const void* q, const void* k_pages, const void* v_pages, void* out,   \
                                                const int* token_seq, const int* token_pos, const int* page_table,    \
                                                int pages_per_seq, int64_t n_tokens, int nq, int nkv, int d,          \
                                                float scale, int window, int value_dim, float softcap,     \
                                                int chunk, int sink, int value_heads, int out_f32,                   \
                                                const float* sink_values, int keep_first, const void* pool_k,         \
                                                const void* pool_v, const int* pool_table, int pool_size,             \
                                                const float* bias, int bias_count, void* stream) {                    \
        const PoolView<T> pool = {(const T*)pool_k, (const T*)pool_v, pool_table, pool_size};                         \
        return attention_generic_launch<T>((const T*)q, (const T*)k_pages, (const T*)v_pages, (T*)out, token_seq,     \
                                           token_pos, page_table, pages_per_seq, n_tokens, nq, nkv, d, scale, window, \
                                           value_dim, softcap, chunk, sink, value_heads, out_f32, sink_values,        \
                                           keep_first, pool, DistanceBias{bias, bias_count}, (cudaStream_t)stream);                                   \
    }                                                                                                                 \
    Q3_EXPORT int q3_value_mix_##SUFFIX(void* rows, int64_t row, int64_t v_off, int width, const float* bias,         \
                                        void* first, int save, float lambda, int64_t n_tokens, void* stream) {        \
        if (n_tokens <= 0) return 0;                                                                                  \
        if (width <= 0 || v_off < 0 || v_off + width > row) return Q3_ERR_BAD_SIZE;                                   \
        constexpr int V = Pack<T>::N;                                                                                 \
        if (width % V == 0 && row % V == 0 && v_off % V == 0 && aligned16(rows) && aligned16(first))                  \
            return launch_flat(value_mix_kernel<T, V>, n_tokens * (width / V), (cudaStream_t)stream, (T*)rows, row,   \
                               v_off, width, bias, (T*)first, save, lambda, n_tokens);                                \
        return launch_flat(value_mix_kernel<T, 1>, n_tokens * width, (cudaStream_t)stream, (T*)rows, row, v_off,      \
                           width, bias, (T*)first, save, lambda, n_tokens);                                           \
    }                                                                                                                 \
    Q3_EXPORT int q3_head_gate_##SUFFIX(void* x, const void* gate, int64_t gate_row, int heads, int vd,               \
                                        int64_t n_tokens, void* stream) {                                             \
        if (n_tokens <= 0) return 0;                                                                                  \
        if (heads <= 0 || vd <= 0) return Q3_ERR_BAD_SIZE;                                                            \
        constexpr int V = Pack<T>::N;                                                                                 \
        if (vd % V == 0 && aligned16(x))                                                                              \
            return launch_flat(head_gate_kernel<T, V>, n_tokens * heads * (vd / V), (cudaStream_t)stream, (T*)x,      \
                               (const T*)gate, gate_row, heads, vd, n_tokens);                                        \
        return launch_flat(head_gate_kernel<T, 1>, n_tokens * heads * vd, (cudaStream_t)stream, (T*)x,                \
                           (const T*)gate, gate_row, heads, vd, n_tokens);                                            \
    }

Q3_ATTENTION_EXPORTS(f32, float)
Q3_ATTENTION_EXPORTS(bf16, bf16)

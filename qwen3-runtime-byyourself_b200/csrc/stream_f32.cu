// Kernels for models whose hidden state between the parts is kept in 32-bit whatever the
// compute type T of the matrix products (float for the 32-bit path, bf16 for serving):
//
//   embedding_scaled : stream[t] = table[ids[t]] * scale                        (T -> float)
//   embedding_sinusoid : the same plus a vector of the token's position p: stream[t, 2i] += sin(p f_i), stream[t, 2i + 1] +=
//                      cos(p f_i).  A frequency is the sum of two floats, so that the angle is right to 32-bit rounding
//                      whatever the position.
//   sandwich_norm    : a branch output y (T) is normalised with weights of its own and added to
//                      the stream, stream += y / rms(y) * w_post, and the sum is normalised for
//                      the next part, out = T(stream / rms(stream) * w_pre): the norm after a
//                      sublayer, the residual sum and the norm before the next sublayer in one
//                      pass over the row.  Either half may be left out (no branch: a plain norm
//                      of the stream; no output: the sum alone).  rms(x) = sqrt(mean(x^2) + eps).
//                      Each norm may be in groups: the row is split into that many equal consecutive parts
//                      and every part is divided by its own rms.
//   concat_cast      : out[t] = T([a[t]; b[t]])  (the input of a product over two streams)
//   gather_rows_norm : rows of the stream picked by index and normalised    (float -> T)
//   normed_sum       : out = T( s_a a / rms(a) * w_a + s_b b / rms(b) * w_b ), two branches of one layer (T)
//   scale_softcap    : x <- cap * tanh(x * scale / cap), or x * scale without a cap (float, in place)
//
// Statistics, weights and sums are 32-bit; only `out` is rounded to T.
#include "common.cuh"

namespace {

template <typename T> __device__ __forceinline__ void load4(const T* p, float (&v)[4]);
template <> __device__ __forceinline__ void load4<float>(const float* p, float (&v)[4]) {
    const float4 r = *reinterpret_cast<const float4*>(p);
    v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
}
template <> __device__ __forceinline__ void load4<bf16>(const bf16* p, float (&v)[4]) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&r.x), b = *reinterpret_cast<const __nv_bfloat162*>(&r.y);
    v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float (&v)[4]);
template <> __device__ __forceinline__ void store4<float>(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, const float (&v)[4]) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 r;
    r.x = *reinterpret_cast<uint32_t*>(&a);
    r.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = r;
}

// ---------------------------------------------------------------- embedding * scale
template <typename T>
__global__ void embedding_scaled_kernel(const int* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out,
                                        int hidden, int vocab, float scale) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    const int id = ids[t];
    const bool ok = id >= 0 && id < vocab;                 // an id outside the table gives a zero row
    const T* src = table + (int64_t)(ok ? id : 0) * hidden;
    for (int c = threadIdx.x; c < hidden; c += blockDim.x) out[t * hidden + c] = ok ? to_f32<T>(src[c]) * scale : 0.0f;
}

// freq: [(hidden + 1) / 2] leading terms, then as many second terms.
template <typename T>
__global__ void embedding_sinusoid_kernel(const int* __restrict__ ids, const int* __restrict__ positions, const T* __restrict__ table,
                                          const float* __restrict__ freq, float* __restrict__ out, int hidden, int vocab, float scale) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t t = blockIdx.x;
    const int id = ids[t], pairs = (hidden + 1) / 2;
    const float p = (float)positions[t];
    const bool ok = id >= 0 && id < vocab;                 // an id outside the table adds nothing to the position's vector
    const T* src = table + (int64_t)(ok ? id : 0) * hidden;
    for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
        // angle = a + rest, a the rounded leading product and rest what it dropped with the second term's part
        const float f = freq[i], a = p * f, rest = fmaf(p, f, -a) + p * freq[pairs + i];
        float s, c, sr, cr;
        sincosf(a, &s, &c);
        sincosf(rest, &sr, &cr);
        const float sine = fmaf(c, sr, s * cr), cosine = fmaf(-s, sr, c * cr);
        float* dst = out + t * hidden + 2 * i;
        dst[0] = (ok ? to_f32<T>(src[2 * i]) * scale : 0.0f) + sine;
        if (2 * i + 1 < hidden) dst[1] = (ok ? to_f32<T>(src[2 * i + 1]) * scale : 0.0f) + cosine;
    }
}

// ---------------------------------------------------------------- norm after a branch + sum + norm before the next
// One block per row; a thread keeps PER groups of four values of the row in registers, so the stream is read and
// written once.  PER = 0: any size, the row walked three times through the cache.  GROUPS: norms over equal parts of
// the row (the statistics of a part are summed by one warp in a fixed order); else over the row as a whole.
struct SandwichArgs {
    int size;
    int parts_post, parts_pre;
    float eps_post, eps_pre;
};

// inv[p] = 1 / rms of part p from the sums of squares of the row's quads (dynamic shared memory: quads, then parts).
__device__ __forceinline__ void part_scales(const float* quad_sq, float* inv, int size, int parts, float eps) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5, per = size / 4 / parts;
    __syncthreads();
    for (int p = warp; p < parts; p += n_warps) {
        float sum = 0.0f;
        for (int i = lane; i < per; i += 32) sum += quad_sq[p * per + i];
        sum = warp_sum(sum);
        if (lane == 0) inv[p] = rsqrtf(sum / (float)(size / parts) + eps);
    }
    __syncthreads();
}
// The same from the row itself, `at(c)` its value at column c.
template <typename F> __device__ __forceinline__ void part_scales_of(F&& at, float* inv, int size, int parts, float eps) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5, per = size / parts;
    __syncthreads();
    for (int p = warp; p < parts; p += n_warps) {
        float sum = 0.0f;
        for (int i = lane; i < per; i += 32) {
            const float v = at(p * per + i);
            sum += v * v;
        }
        sum = warp_sum(sum);
        if (lane == 0) inv[p] = rsqrtf(sum / (float)per + eps);
    }
    __syncthreads();
}

template <typename T, int PER, bool GROUPS>
__global__ void sandwich_norm_kernel(float* __restrict__ stream, const T* __restrict__ branch, const float* __restrict__ w_post,
                                     const float* __restrict__ w_pre, T* __restrict__ out, const SandwichArgs args) {
    __shared__ float scratch[33];
    extern __shared__ float parts_s[];
    pdl_launch_dependents();
    pdl_wait();
    const int size = args.size;
    const int64_t row = blockIdx.x;
    float* xr = stream + row * size;
    const T* yr = branch ? branch + row * size : nullptr;
    T* outr = out ? out + row * size : nullptr;
    if constexpr (PER > 0) {
        float* quad_sq = parts_s;                          // [size / 4]
        float* inv_s = parts_s + size / 4;                 // [parts]
        float x[PER][4], y[PER][4];
        float sq = 0.0f;
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int c = (p * blockDim.x + threadIdx.x) * 4;
            if (c < size) {
                load4<float>(xr + c, x[p]);
                if (yr) {
                    load4<T>(yr + c, y[p]);
                    if constexpr (GROUPS) quad_sq[c >> 2] = (y[p][0] * y[p][0] + y[p][1] * y[p][1]) + (y[p][2] * y[p][2] + y[p][3] * y[p][3]);
#pragma unroll
                    for (int i = 0; i < 4; ++i) sq += y[p][i] * y[p][i];
                }
            }
        }
        if (yr) {
            float inv = 0.0f;
            if constexpr (GROUPS) part_scales(quad_sq, inv_s, size, args.parts_post, args.eps_post);
            else inv = rsqrtf(block_sum(sq, scratch) / (float)size + args.eps_post);
#pragma unroll
            for (int p = 0; p < PER; ++p) {
                const int c = (p * blockDim.x + threadIdx.x) * 4;
                if (c < size) {
                    if constexpr (GROUPS) inv = inv_s[c / (size / args.parts_post)];
                    float w[4];
                    load4<float>(w_post + c, w);
#pragma unroll
                    for (int i = 0; i < 4; ++i) x[p][i] += y[p][i] * inv * w[i];
                    store4<float>(xr + c, x[p]);
                }
            }
        }
        if (outr == nullptr) return;
        sq = 0.0f;
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int c = (p * blockDim.x + threadIdx.x) * 4;
            if (c < size) {
                if constexpr (GROUPS) quad_sq[c >> 2] = (x[p][0] * x[p][0] + x[p][1] * x[p][1]) + (x[p][2] * x[p][2] + x[p][3] * x[p][3]);
#pragma unroll
                for (int i = 0; i < 4; ++i) sq += x[p][i] * x[p][i];
            }
        }
        float inv = 0.0f;
        if constexpr (GROUPS) part_scales(quad_sq, inv_s, size, args.parts_pre, args.eps_pre);
        else inv = rsqrtf(block_sum(sq, scratch) / (float)size + args.eps_pre);
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int c = (p * blockDim.x + threadIdx.x) * 4;
            if (c < size) {
                if constexpr (GROUPS) inv = inv_s[c / (size / args.parts_pre)];
                float w[4], v[4];
                load4<float>(w_pre + c, w);
#pragma unroll
                for (int i = 0; i < 4; ++i) v[i] = x[p][i] * inv * w[i];
                store4<T>(outr + c, v);
            }
        }
    } else {
        float* inv_s = parts_s;                            // [parts]
        if (yr) {
            const int per = size / args.parts_post;
            part_scales_of([&](int c) { return to_f32<T>(yr[c]); }, inv_s, size, args.parts_post, args.eps_post);
            for (int c = threadIdx.x; c < size; c += blockDim.x) xr[c] += to_f32<T>(yr[c]) * inv_s[c / per] * w_post[c];
        }
        if (outr == nullptr) return;
        const int per = size / args.parts_pre;
        part_scales_of([&](int c) { return xr[c]; }, inv_s, size, args.parts_pre, args.eps_pre);
        for (int c = threadIdx.x; c < size; c += blockDim.x) outr[c] = from_f32<T>(xr[c] * inv_s[c / per] * w_pre[c]);
    }
}

template <typename T>
int sandwich_norm_launch(float* stream, const T* branch, const float* w_post, const float* w_pre, T* out, int64_t rows, int size,
                         float eps_post, float eps_pre, int parts_post, int parts_pre, cudaStream_t s) {
    if (rows <= 0) return 0;
    if (size <= 0 || (branch != nullptr) != (w_post != nullptr) || (out != nullptr) != (w_pre != nullptr)) return Q3_ERR_BAD_SIZE;
    if (parts_post <= 0 || parts_pre <= 0 || size % parts_post != 0 || size % parts_pre != 0) return Q3_ERR_BAD_SIZE;
    if (rows > 0x7fffffffLL) return Q3_ERR_TOO_LARGE;
    const bool grouped = parts_post > 1 || parts_pre > 1;
    const bool vec = size % 4 == 0 && (!grouped || ((size / parts_post) % 4 == 0 && (size / parts_pre) % 4 == 0)) && aligned16(stream) &&
                     (branch == nullptr || aligned16(branch)) && (out == nullptr || aligned16(out)) &&
                     (w_post == nullptr || aligned16(w_post)) && (w_pre == nullptr || aligned16(w_pre));
    const int groups = size / 4, parts = parts_post > parts_pre ? parts_post : parts_pre;
    const SandwichArgs args = {size, parts_post, parts_pre, eps_post, eps_pre};
    auto launch = [&](auto kernel, int threads, size_t smem) {
        return (int)q3_launch(kernel, dim3((unsigned)rows), dim3(threads), smem, s, stream, branch, w_post, w_pre, out, args);
    };
    if (vec && groups <= 2048) {
        const int per = groups <= 256 ? 1 : (groups <= 512 ? 2 : (groups <= 1024 ? 4 : 8));
        const int threads = ((groups + per - 1) / per + 31) / 32 * 32;
        const size_t smem = grouped ? (size_t)(groups + parts) * sizeof(float) : 0;
#define Q3_SANDWICH(PER) return grouped ? launch(sandwich_norm_kernel<T, PER, true>, threads, smem) : launch(sandwich_norm_kernel<T, PER, false>, threads, 0)
        if (per == 1) Q3_SANDWICH(1);
        if (per == 2) Q3_SANDWICH(2);
        if (per == 4) Q3_SANDWICH(4);
        Q3_SANDWICH(8);
#undef Q3_SANDWICH
    }
    if (parts > 8192) return Q3_ERR_TOO_LARGE;
    return launch(sandwich_norm_kernel<T, 0, true>, size >= 1024 ? 512 : 128, (size_t)parts * sizeof(float));
}

// ---------------------------------------------------------------- two normed branches in one sum
// Two sums over a block at once; `scratch` holds 66 floats.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = (blockDim.x + 31) >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    if (lane == 0) {
        scratch[warp] = a;
        scratch[33 + warp] = b;
    }
    __syncthreads();
    a = warp_sum(lane < n_warps ? scratch[lane] : 0.0f);        // every warp adds them up for itself
    b = warp_sum(lane < n_warps ? scratch[33 + lane] : 0.0f);
    return make_float2(a, b);
}

// One block per row.  PER > 0: a thread keeps PER groups of four values of both rows in registers.
template <typename T, int PER>
__global__ void normed_sum_kernel(const T* __restrict__ a, const T* __restrict__ b, const float* __restrict__ w_a,
                                  const float* __restrict__ w_b, float s_a, float s_b, float eps, T* __restrict__ out, int size) {
    __shared__ float scratch[66];
    pdl_launch_dependents();
    pdl_wait();
    const T* ar = a + (int64_t)blockIdx.x * size;
    const T* br = b + (int64_t)blockIdx.x * size;
    T* outr = out + (int64_t)blockIdx.x * size;
    float sq_a = 0.0f, sq_b = 0.0f;
    if constexpr (PER > 0) {
        float x[PER][4], y[PER][4];
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int c = (p * blockDim.x + threadIdx.x) * 4;
            if (c < size) {
                load4<T>(ar + c, x[p]);
                load4<T>(br + c, y[p]);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    sq_a += x[p][i] * x[p][i];
                    sq_b += y[p][i] * y[p][i];
                }
            }
        }
        const float2 sums = block_sum2(sq_a, sq_b, scratch);
        const float inv_a = s_a * rsqrtf(sums.x / (float)size + eps), inv_b = s_b * rsqrtf(sums.y / (float)size + eps);
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const int c = (p * blockDim.x + threadIdx.x) * 4;
            if (c < size) {
                float wa[4], wb[4], v[4];
                load4<float>(w_a + c, wa);
                load4<float>(w_b + c, wb);
#pragma unroll
                for (int i = 0; i < 4; ++i) v[i] = x[p][i] * inv_a * wa[i] + y[p][i] * inv_b * wb[i];
                store4<T>(outr + c, v);
            }
        }
    } else {
        for (int c = threadIdx.x; c < size; c += blockDim.x) {
            const float x = to_f32<T>(ar[c]), y = to_f32<T>(br[c]);
            sq_a += x * x;
            sq_b += y * y;
        }
        const float2 sums = block_sum2(sq_a, sq_b, scratch);
        const float inv_a = s_a * rsqrtf(sums.x / (float)size + eps), inv_b = s_b * rsqrtf(sums.y / (float)size + eps);
        for (int c = threadIdx.x; c < size; c += blockDim.x)
            outr[c] = from_f32<T>(to_f32<T>(ar[c]) * inv_a * w_a[c] + to_f32<T>(br[c]) * inv_b * w_b[c]);
    }
}

template <typename T>
int normed_sum_launch(const T* a, const T* b, const float* w_a, const float* w_b, float s_a, float s_b, float eps, T* out, int64_t rows,
                      int size, cudaStream_t s) {
    if (rows <= 0) return 0;
    if (size <= 0 || w_a == nullptr || w_b == nullptr) return Q3_ERR_BAD_SIZE;
    if (rows > 0x7fffffffLL) return Q3_ERR_TOO_LARGE;
    auto launch = [&](auto kernel, int threads) {
        return (int)q3_launch(kernel, dim3((unsigned)rows), dim3(threads), 0, s, a, b, w_a, w_b, s_a, s_b, eps, out, size);
    };
    const int groups = size / 4;
    if (size % 4 == 0 && groups <= 2048 && aligned16(a) && aligned16(b) && aligned16(w_a) && aligned16(w_b) && aligned16(out)) {
        const int per = groups <= 256 ? 1 : (groups <= 512 ? 2 : (groups <= 1024 ? 4 : 8));
        const int threads = ((groups + per - 1) / per + 31) / 32 * 32;
        if (per == 1) return launch(normed_sum_kernel<T, 1>, threads);
        if (per == 2) return launch(normed_sum_kernel<T, 2>, threads);
        if (per == 4) return launch(normed_sum_kernel<T, 4>, threads);
        return launch(normed_sum_kernel<T, 8>, threads);
    }
    return launch(normed_sum_kernel<T, 0>, size >= 1024 ? 512 : 128);
}

// ---------------------------------------------------------------- [a; b] in the compute type
// Four values a thread where the rows allow 16-byte reads.
template <typename T>
__global__ void concat_cast_vec_kernel(const float* __restrict__ a, const float* __restrict__ b, T* __restrict__ out, int64_t rows,
                                       int size) {
    pdl_launch_dependents();
    pdl_wait();
    const int groups = size / 4;
    const int64_t total = rows * 2 * groups;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = i / (2 * groups);
        const int g = (int)(i % (2 * groups));
        float v[4];
        load4<float>((g < groups ? a + r * size : b + r * size - size) + 4 * g, v);
        store4<T>(out + r * 2 * size + 4 * g, v);
    }
}

template <typename T>
__global__ void concat_cast_kernel(const float* __restrict__ a, const float* __restrict__ b, T* __restrict__ out, int64_t rows,
                                   int size) {
    pdl_launch_dependents();
    pdl_wait();
    const int64_t total = rows * 2 * size;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (int64_t)gridDim.x * blockDim.x) {
        const int64_t r = i / (2 * size);
        const int c = (int)(i % (2 * size));
        out[i] = from_f32<T>(c < size ? a[r * size + c] : b[r * size + c - size]);
    }
}

// ---------------------------------------------------------------- picked rows, normalised
template <typename T>
__global__ void gather_rows_norm_kernel(const float* __restrict__ stream, const int* __restrict__ idx, const float* __restrict__ w,
                                        T* __restrict__ out, int size, float eps, int parts) {
    __shared__ float scratch[33];
    extern __shared__ float inv_s[];                       // [parts] if there are several
    pdl_launch_dependents();
    pdl_wait();
    const float* xr = stream + (int64_t)idx[blockIdx.x] * size;
    float inv = 0.0f;
    const int per = size / parts;
    if (parts == 1) {
        float sq = 0.0f;
        for (int c = threadIdx.x; c < size; c += blockDim.x) sq += xr[c] * xr[c];
        inv = rsqrtf(block_sum(sq, scratch) / (float)size + eps);
    } else {
        part_scales_of([&](int c) { return xr[c]; }, inv_s, size, parts, eps);
    }
    for (int c = threadIdx.x; c < size; c += blockDim.x)
        out[(int64_t)blockIdx.x * size + c] = from_f32<T>(xr[c] * (parts == 1 ? inv : inv_s[c / per]) * w[c]);
}

// ---------------------------------------------------------------- scale and smooth cap, in place
__global__ void scale_softcap_kernel(float* __restrict__ x, int64_t n, float scale, float cap) {
    pdl_launch_dependents();
    pdl_wait();
    const float inv = cap > 0.0f ? 1.0f / cap : 0.0f;
    for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
        const float v = x[i] * scale;
        x[i] = cap > 0.0f ? cap * tanhf(v * inv) : v;
    }
}

static unsigned grid_for(int64_t work, int threads) {
    int64_t blocks = (work + threads - 1) / threads;
    const int64_t resident = (int64_t)q3_device_sm_count() * 8;
    return (unsigned)(blocks > resident ? resident : (blocks < 1 ? 1 : blocks));
}

}  // namespace

#define Q3_STREAM_EXPORTS(SUFFIX, T)                                                                                     \
    Q3_EXPORT int q3_embedding_sinusoid_##SUFFIX(const int* ids, const int* positions, const void* table, const float* freq, \
                                                 float* out, int64_t n_tokens, int hidden, int vocab, float scale,        \
                                                 void* stream) {                                                          \
        if (n_tokens <= 0) return 0;                                                                                      \
        if (hidden <= 0 || vocab <= 0) return Q3_ERR_BAD_SIZE;                                                            \
        if (n_tokens > 0x7fffffffLL) return Q3_ERR_TOO_LARGE;                                                             \
        return (int)q3_launch(embedding_sinusoid_kernel<T>, dim3((unsigned)n_tokens), dim3(hidden >= 512 ? 256 : 64), 0,  \
                              (cudaStream_t)stream, ids, positions, (const T*)table, freq, out, hidden, vocab, scale);    \
    }                                                                                                                     \
    Q3_EXPORT int q3_embedding_scaled_##SUFFIX(const int* ids, const void* table, float* out, int64_t n_tokens, int hidden, \
                                               int vocab, float scale, void* stream) {                                  \
        if (n_tokens <= 0) return 0;                                                                                     \
        if (hidden <= 0 || n_tokens > 0x7fffffffLL) return Q3_ERR_BAD_SIZE;                                              \
        return (int)q3_launch(embedding_scaled_kernel<T>, dim3((unsigned)n_tokens), dim3(hidden >= 1024 ? 256 : 128), 0, \
                              (cudaStream_t)stream, ids, (const T*)table, out, hidden, vocab, scale);                    \
    }                                                                                                                    \
    Q3_EXPORT int q3_sandwich_norm_##SUFFIX(float* stream_rows, const void* branch, const float* w_post, const float* w_pre, \
                                            void* out, int64_t rows, int size, float eps_post, float eps_pre,           \
                                            int parts_post, int parts_pre, void* stream) {                               \
        return sandwich_norm_launch<T>(stream_rows, (const T*)branch, w_post, w_pre, (T*)out, rows, size, eps_post,      \
                                       eps_pre, parts_post, parts_pre, (cudaStream_t)stream);                            \
    }                                                                                                                    \
    Q3_EXPORT int q3_normed_sum_##SUFFIX(const void* a, const void* b, const float* w_a, const float* w_b, float s_a,    \
                                         float s_b, float eps, void* out, int64_t rows, int size, void* stream) {        \
        return normed_sum_launch<T>((const T*)a, (const T*)b, w_a, w_b, s_a, s_b, eps, (T*)out, rows, size,              \
                                    (cudaStream_t)stream);                                                               \
    }                                                                                                                    \
    Q3_EXPORT int q3_concat_cast_##SUFFIX(const float* a, const float* b, void* out, int64_t rows, int size, void* stream) { \
        if (rows <= 0) return 0;                                                                                         \
        if (size <= 0) return Q3_ERR_BAD_SIZE;                                                                           \
        if (size % 4 == 0 && aligned16(a) && aligned16(b) && aligned16(out))                                             \
            return (int)q3_launch(concat_cast_vec_kernel<T>, dim3(grid_for(rows * 2 * (size / 4), 256)), dim3(256), 0,   \
                                  (cudaStream_t)stream, a, b, (T*)out, rows, size);                                      \
        return (int)q3_launch(concat_cast_kernel<T>, dim3(grid_for(rows * 2 * size, 256)), dim3(256), 0,                 \
                              (cudaStream_t)stream, a, b, (T*)out, rows, size);                                          \
    }                                                                                                                    \
    Q3_EXPORT int q3_gather_rows_norm_##SUFFIX(const float* stream_rows, const int* idx, const float* w, void* out,      \
                                               int64_t rows, int size, float eps, int parts, void* stream) {             \
        if (rows <= 0) return 0;                                                                                         \
        if (size <= 0 || rows > 0x7fffffffLL || parts <= 0 || size % parts != 0 || parts > 8192) return Q3_ERR_BAD_SIZE; \
        return (int)q3_launch(gather_rows_norm_kernel<T>, dim3((unsigned)rows), dim3(size >= 1024 ? 256 : 128),          \
                              parts > 1 ? (size_t)parts * sizeof(float) : 0, (cudaStream_t)stream, stream_rows, idx, w,  \
                              (T*)out, size, eps, parts);                                                                \
    }

Q3_STREAM_EXPORTS(f32, float)
Q3_STREAM_EXPORTS(bf16, bf16)

Q3_EXPORT int q3_scale_softcap_f32(float* x, int64_t n, float scale, float cap, void* stream) {
    if (n <= 0) return 0;
    return (int)q3_launch(scale_softcap_kernel, dim3(grid_for(n, 256)), dim3(256), 0, (cudaStream_t)stream, x, n, scale, cap);
}

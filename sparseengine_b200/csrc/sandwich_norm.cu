// Norms before and after a sublayer over a 32-bit residual stream, as one kernel between two sublayers:
//
//     c   = y                                                    (one result)
//         | s0 rms(y0) w0 + s1 rms(y1) w1                        (two results side by side, each normed by itself)
//     c   = rms(c) post_w                                        (the norm after the sublayer, optional)
//     x   = stream + c                                           (32-bit, stored back; the stream is optional)
//     out = rms(x) next_w, rounded to the activation type        (the norm before the next sublayer; without next_w: x)
//
// with rms(v) = v / sqrt(mean(v^2) + eps).  Everything between the loads and the last rounding is 32-bit.  One block
// per row.  `rows` (optional) names the stream's and the results' row of every output row: the norm before a model's
// head reads only the rows that are asked for (the stream is then not stored).
//
// Rows of up to 16,384 elements (a multiple of 8, 16-byte aligned) stay in registers, each input is read once and a
// reduction is one barrier; weights are fetched before the kernel ahead has ended.  Other rows go through shared memory.
#include "common.cuh"

namespace se {
namespace sandwich {

struct Args {
    float* stream;               // [*, hidden] or nullptr
    const void *y0, *y1;         // [*, hidden]; y1 nullptr: one result; y0 nullptr: none
    const void *w0, *w1;         // weights of the two results' own norms
    float s0, s1, eps_pair;
    const void* post_w;          // nullptr: no norm after the sublayer
    float eps_post;
    const void* next_w;          // nullptr: no norm
    float eps_next;
    void* out;                   // [rows, hidden] or nullptr
    const int* rows;             // nullptr: row i
    int num_rows_in;             // rows of the stream and the results (bounds `rows`)
    int hidden, store;
};

constexpr int kMaxThreads = 512;

// Eight neighbours as they lie in memory.
template <typename T> struct Raw8;
template <> struct Raw8<__nv_bfloat16> {
    uint4 r;
    __device__ __forceinline__ void load(const __nv_bfloat16* p) { r = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void get(float* v) const {
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 f = __bfloat1622float2(h[i]);
            v[2 * i] = f.x;
            v[2 * i + 1] = f.y;
        }
    }
};
template <> struct Raw8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) {
        a = *reinterpret_cast<const float4*>(p);
        b = *reinterpret_cast<const float4*>(p + 4);
    }
    __device__ __forceinline__ void get(float* v) const {
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
};

// Sums over the block with one barrier: every warp leaves its part in `part` (a buffer of its own per sum), every
// thread adds them up in the same order.
__device__ __forceinline__ float sum1(float v, float* part) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    v = warp_sum(v);
    if (lane == 0) part[warp] = v;
    __syncthreads();
    float t = 0.f;
    for (int i = 0; i < warps; ++i) t += part[i];
    return t;
}
__device__ __forceinline__ float2 sum2(float a, float b, float2* part) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    if (lane == 0) part[warp] = make_float2(a, b);
    __syncthreads();
    float2 t = make_float2(0.f, 0.f);
    for (int i = 0; i < warps; ++i) { t.x += part[i].x; t.y += part[i].y; }
    return t;
}

// CH: chunks of 8 elements a thread keeps; NY: results (0, 1, 2).
template <typename T, int CH, int NY>
__global__ void __launch_bounds__(kMaxThreads)
sandwich_norm_kernel(const Args p) {
    __shared__ float2 part_pair[kMaxThreads / 32];
    __shared__ float part_post[kMaxThreads / 32], part_next[kMaxThreads / 32];
    const int hidden = p.hidden, step = blockDim.x * 8, i0 = threadIdx.x * 8;
    const T *w0 = (const T*)p.w0, *w1 = (const T*)p.w1, *post_w = (const T*)p.post_w, *next_w = (const T*)p.next_w;
    grid_dependency_trigger();
    Raw8<T> w0r[NY == 2 ? CH : 1], w1r[NY == 2 ? CH : 1], postr[NY ? CH : 1], nextr[CH];
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        const int i = i0 + k * step;
        if (i >= hidden) break;
        if (NY == 2) { w0r[k].load(w0 + i); w1r[k].load(w1 + i); }
        if (NY && post_w != nullptr) postr[k].load(post_w + i);
        if (next_w != nullptr) nextr[k].load(next_w + i);
    }
    grid_dependency_wait();
    int row = blockIdx.x;
    if (p.rows != nullptr) {
        row = p.rows[blockIdx.x];
        if ((unsigned)row >= (unsigned)p.num_rows_in) return;
    }
    const size_t base = (size_t)row * hidden;
    float x[CH][8], c[CH][8];
    Raw8<T> y0r[NY ? CH : 1], y1r[NY == 2 ? CH : 1];
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        const int i = i0 + k * step;
#pragma unroll
        for (int j = 0; j < 8; ++j) x[k][j] = c[k][j] = 0.f;
        if (i < hidden) {
            if (NY) y0r[k].load((const T*)p.y0 + base + i);
            if (NY == 2) y1r[k].load((const T*)p.y1 + base + i);
            if (p.stream != nullptr) load8(p.stream + base + i, x[k]);
        }
    }
    if (NY == 1) {
#pragma unroll
        for (int k = 0; k < CH; ++k)
            if (i0 + k * step < hidden) y0r[k].get(c[k]);
    }
    if (NY == 2) {
        float sa = 0.f, sb = 0.f;
#pragma unroll
        for (int k = 0; k < CH; ++k) {
            if (i0 + k * step >= hidden) break;
            float a[8], b[8];
            y0r[k].get(a);
            y1r[k].get(b);
#pragma unroll
            for (int j = 0; j < 8; ++j) { sa += a[j] * a[j]; sb += b[j] * b[j]; }
        }
        const float2 ss = sum2(sa, sb, part_pair);
        const float ra = p.s0 / sqrtf(ss.x / (float)hidden + p.eps_pair), rb = p.s1 / sqrtf(ss.y / (float)hidden + p.eps_pair);
#pragma unroll
        for (int k = 0; k < CH; ++k) {
            if (i0 + k * step >= hidden) break;
            float a[8], b[8], wa[8], wb[8];
            y0r[k].get(a);
            y1r[k].get(b);
            w0r[k].get(wa);
            w1r[k].get(wb);
#pragma unroll
            for (int j = 0; j < 8; ++j) c[k][j] = a[j] * ra * wa[j] + b[j] * rb * wb[j];
        }
    }
    if (NY && post_w != nullptr) {
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < CH; ++k)
#pragma unroll
            for (int j = 0; j < 8; ++j) s += c[k][j] * c[k][j];
        const float r = 1.0f / sqrtf(sum1(s, part_post) / (float)hidden + p.eps_post);
#pragma unroll
        for (int k = 0; k < CH; ++k) {
            if (i0 + k * step >= hidden) break;
            float wp[8];
            postr[k].get(wp);
#pragma unroll
            for (int j = 0; j < 8; ++j) c[k][j] *= r * wp[j];
        }
    }
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        const int i = i0 + k * step;
        if (i >= hidden) break;
        if (NY) {
#pragma unroll
            for (int j = 0; j < 8; ++j) x[k][j] += c[k][j];
        }
        if (p.store) store8(p.stream + base + i, x[k]);
    }
    if (p.out == nullptr) return;
    float r = 1.f;
    if (next_w != nullptr) {
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < CH; ++k)
#pragma unroll
            for (int j = 0; j < 8; ++j) s += x[k][j] * x[k][j];
        r = 1.0f / sqrtf(sum1(s, part_next) / (float)hidden + p.eps_next);
    }
    T* out = (T*)p.out + (size_t)blockIdx.x * hidden;
#pragma unroll
    for (int k = 0; k < CH; ++k) {
        const int i = i0 + k * step;
        if (i >= hidden) break;
        if (next_w != nullptr) {
            float wn[8];
            nextr[k].get(wn);
#pragma unroll
            for (int j = 0; j < 8; ++j) x[k][j] *= r * wn[j];
        }
        store8(out + i, x[k]);
    }
}

// Any width: the row in shared memory, element by element.
template <typename T>
__global__ void sandwich_norm_any_kernel(const Args p) {
    extern __shared__ __align__(16) float xs[];
    __shared__ float scratch[33];
    grid_dependency_trigger();
    grid_dependency_wait();
    int row = blockIdx.x;
    if (p.rows != nullptr) {
        row = p.rows[blockIdx.x];
        if ((unsigned)row >= (unsigned)p.num_rows_in) return;
    }
    const int hidden = p.hidden;
    const size_t base = (size_t)row * hidden;
    const T *y0 = p.y0 != nullptr ? (const T*)p.y0 + base : nullptr, *y1 = p.y1 != nullptr ? (const T*)p.y1 + base : nullptr;
    const T *w0 = (const T*)p.w0, *w1 = (const T*)p.w1, *post_w = (const T*)p.post_w, *next_w = (const T*)p.next_w;
    auto inv_rms = [&](float ss, float eps) { return 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps); };
    // every thread reads back the elements of the row that it wrote itself
    if (y0 != nullptr) {
        float ra = 1.f, rb = 1.f, ss = 0.f;
        if (y1 != nullptr) {
            float sa = 0.f, sb = 0.f;
            for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
                const float a = to_float(y0[i]), b = to_float(y1[i]);
                sa += a * a;
                sb += b * b;
            }
            ra = p.s0 * inv_rms(sa, p.eps_pair);
            rb = p.s1 * inv_rms(sb, p.eps_pair);
        }
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
            float v = to_float(y0[i]);
            if (y1 != nullptr) v = v * ra * to_float(w0[i]) + to_float(y1[i]) * rb * to_float(w1[i]);
            xs[i] = v;
            ss += v * v;
        }
        const float r = post_w != nullptr ? inv_rms(ss, p.eps_post) : 1.f;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x)
            xs[i] = xs[i] * r * (post_w != nullptr ? to_float(post_w[i]) : 1.f) + (p.stream != nullptr ? p.stream[base + i] : 0.f);
    } else {
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) xs[i] = p.stream[base + i];
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = xs[i];
        ss += v * v;
        if (p.store) p.stream[base + i] = v;
    }
    if (p.out == nullptr) return;
    const float r = next_w != nullptr ? inv_rms(ss, p.eps_next) : 1.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x)
        ((T*)p.out)[(size_t)blockIdx.x * hidden + i] = from_float<T>(xs[i] * r * (next_w != nullptr ? to_float(next_w[i]) : 1.f));
}

template <typename T, int NY>
static cudaError_t launch(const Args& a, int rows, bool vec, cudaStream_t stream) {
    const int chunks = a.hidden / 8;
    if (vec && chunks <= 4 * kMaxThreads) {
        // few rows, and two results: as many threads as there are chunks; many rows of one result: two chunks a thread
        const int want = NY < 2 && rows >= 1024 && chunks >= 256 ? (chunks + 1) / 2 : chunks;
        int threads = (want + 31) / 32 * 32;
        if (threads > kMaxThreads) threads = kMaxThreads;
        const int ch = (chunks + threads - 1) / threads;
        if (ch == 1) return SE_LAUNCH_DEPENDENT("norm", (sandwich_norm_kernel<T, 1, NY>), dim3(rows), dim3(threads), 0, stream, a);
        if (ch == 2) return SE_LAUNCH_DEPENDENT("norm", (sandwich_norm_kernel<T, 2, NY>), dim3(rows), dim3(threads), 0, stream, a);
        return SE_LAUNCH_DEPENDENT("norm", (sandwich_norm_kernel<T, 4, NY>), dim3(rows), dim3(threads), 0, stream, a);
    }
    const size_t smem = (size_t)a.hidden * sizeof(float);
    if (smem > 40 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(sandwich_norm_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    return SE_LAUNCH_DEPENDENT("norm", sandwich_norm_any_kernel<T>, dim3(rows), dim3(a.hidden >= 1024 ? 256 : 128), smem, stream, a);
}

}  // namespace sandwich
}  // namespace se

extern "C" int se_sandwich_norm_max_width() { return 200 * 1024 / (int)sizeof(float); }

// dtype: the type of the results, the weights and `out`.  y1 == nullptr: one result (w0, w1, s0, s1, eps_pair unused).
extern "C" int se_sandwich_norm(float* stream_, const void* y0, const void* y1, const void* w0, const void* w1, float s0, float s1,
                                float eps_pair, const void* post_w, float eps_post, const void* next_w, float eps_next, void* out,
                                const int* rows_index, int rows_in, int rows, int hidden, int store, int dtype, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (hidden <= 0 || hidden > se_sandwich_norm_max_width()) return SE_ERR_UNSUPPORTED;
    if (y0 == nullptr && (y1 != nullptr || post_w != nullptr || stream_ == nullptr)) return SE_ERR_ARGUMENT;
    if (y1 != nullptr && (w0 == nullptr || w1 == nullptr)) return SE_ERR_ARGUMENT;
    if (store && (stream_ == nullptr || rows_index != nullptr)) return SE_ERR_ARGUMENT;
    if (!store && out == nullptr) return 0;
    const se::sandwich::Args a{stream_, y0, y1, w0, w1, s0, s1, eps_pair, post_w, eps_post, next_w, eps_next, out, rows_index, rows_in, hidden, store};
    uintptr_t bits = 0;
    for (const void* q : {(const void*)stream_, y0, y1, w0, w1, post_w, next_w, (const void*)out}) bits |= reinterpret_cast<uintptr_t>(q);
    const bool vec = hidden % 8 == 0 && (bits & 15) == 0;
    SE_DISPATCH_DTYPE(dtype, T, {
        const cudaError_t e = y0 == nullptr ? se::sandwich::launch<T, 0>(a, rows, vec, stream)
                              : y1 == nullptr ? se::sandwich::launch<T, 1>(a, rows, vec, stream)
                                              : se::sandwich::launch<T, 2>(a, rows, vec, stream);
        if (e != cudaSuccess) return (int)e;
    });
    SE_LAUNCH_CHECK();
}

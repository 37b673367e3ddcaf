// A gated recurrence whose gates read the current token only (minGRU).  Per channel, with the projections
// z', u', g of a token and biases b_z, b_u:
//
//     z = sigmoid(z' + b_z),   u = u' + b_u,   c = u + 1/2 (u >= 0) or sigmoid(u) (u < 0)
//     S <- (1 - z) S + z c,    y = S * silu(g)
//
// Everything between the projections and y is 32-bit; the state is one 32-bit row of `width` per request.
// A projection row is [z' | u' | g], each `width` wide; cu_q gives each entry's tokens and seq_rows its state row.
//
// Two kernels.  `scan`: a thread per channel pair walks an entry's tokens (single tokens, short pieces).
// `chunk`: prompt portions.  Since S after a run of tokens is A S + B with A = prod (1 - z), runs compose, so the
// tokens are dealt out: a cluster of up to eight CTAs takes 64 channels of one entry, each CTA 128 tokens at a time,
// each of its warps 16 of them.  A warp computes its tokens' (1 - z, z c) once, keeps them in registers and folds
// them to one pair (A, B) per channel; the pairs travel through shared memory inside the CTA and through
// distributed shared memory between the CTAs; then every warp knows the state before its first token and walks its
// tokens from registers.  Each input is read from memory once.
#include "common.cuh"
#include <cooperative_groups.h>

namespace se {
namespace gru {

namespace cg = cooperative_groups;

constexpr int kWarps = 8;
constexpr int kTokens = 16;                  // tokens of a warp at a time
constexpr int kTile = kWarps * kTokens;      // tokens of a CTA at a time
constexpr int kChannels = 64;                // channels of a CTA: two per lane
constexpr int kMaxCluster = 8;

// 16-bit activations take the special-function unit's exponential and reciprocal (a few units in the last place of
// 32-bit; beyond their range the results are 0 and 1, as they should be)
template <typename T> __device__ __forceinline__ float sigmoid(float x) {
    if (sizeof(T) != 2) return 1.f / (1.f + expf(-x));
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * -1.4426950408889634f));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
    return r;
}
template <typename T> __device__ __forceinline__ void cell(float zl, float u, float& keep, float& add) {
    const float z = sigmoid<T>(zl);
    keep = 1.f - z;
    add = z * (u >= 0.f ? u + 0.5f : sigmoid<T>(u));
}
template <typename T> __device__ __forceinline__ float silu(float x) { return x * sigmoid<T>(x); }

__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const __nv_bfloat16* p) {
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void store2(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
__device__ __forceinline__ void store2(__nv_bfloat16* p, float2 v) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y);
}
// the channels c and c + 1 of a row (PAIR: both exist and the pair can be read in one piece)
template <bool PAIR, typename T> __device__ __forceinline__ float2 read2(const T* row, int c, int width) {
    if (PAIR) return load2(row + c);
    return make_float2(to_float(row[c]), c + 1 < width ? to_float(row[c + 1]) : 0.f);
}
template <bool PAIR, typename T> __device__ __forceinline__ void write2(T* row, int c, int width, float2 v) {
    if (PAIR) { store2(row + c, v); return; }
    row[c] = from_float<T>(v.x);
    if (c + 1 < width) row[c + 1] = from_float<T>(v.y);
}

// the same as stored (a register for a pair of bfloat16), to be unpacked later
template <typename T> struct Stored { using type = float2; };
template <> struct Stored<__nv_bfloat16> { using type = __nv_bfloat162; };
template <bool PAIR> __device__ __forceinline__ float2 read_stored(const float* row, int c, int width) { return read2<PAIR>(row, c, width); }
template <bool PAIR> __device__ __forceinline__ __nv_bfloat162 read_stored(const __nv_bfloat16* row, int c, int width) {
    if (PAIR) return *reinterpret_cast<const __nv_bfloat162*>(row + c);
    return __halves2bfloat162(row[c], c + 1 < width ? row[c + 1] : row[c]);
}
__device__ __forceinline__ float2 unpack(float2 v) { return v; }
__device__ __forceinline__ float2 unpack(__nv_bfloat162 v) { return __bfloat1622float2(v); }

template <typename T, bool PAIR>
__global__ void __launch_bounds__(128)
min_gru_scan_kernel(const T* proj, int pitch, const float* __restrict__ bias, float* state, long long state_stride,
                    const int* __restrict__ cu_q, const int* __restrict__ seq_rows, T* out, int width) {
    grid_dependency_trigger();
    const int c = 2 * (blockIdx.x * blockDim.x + threadIdx.x);
    float2 bz, bu;
    if (c < width) { bz = read2<false>(bias, c, width); bu = read2<false>(bias + width, c, width); }
    grid_dependency_wait();
    if (c >= width) return;
    const int entry = blockIdx.y;
    const int t1 = cu_q[entry + 1];
    float* srow = state + (size_t)seq_rows[entry] * state_stride;
    float2 s = read2<false>(srow, c, width);
    for (int t = cu_q[entry]; t < t1; ++t) {
        const T* row = proj + (size_t)t * pitch;
        const float2 z = read2<PAIR>(row, c, width), u = read2<PAIR>(row + width, c, width), g = read2<PAIR>(row + 2 * width, c, width);
        float keep, add;
        cell<T>(z.x + bz.x, u.x + bu.x, keep, add);
        s.x = keep * s.x + add;
        cell<T>(z.y + bz.y, u.y + bu.y, keep, add);
        s.y = keep * s.y + add;
        write2<PAIR>(out + (size_t)t * width, c, width, make_float2(s.x * silu<T>(g.x), s.y * silu<T>(g.y)));
    }
    write2<false>(srow, c, width, s);
}

template <typename T, bool PAIR>
__global__ void __launch_bounds__(32 * kWarps, 2)
min_gru_chunk_kernel(const T* __restrict__ proj, int pitch, const float* __restrict__ bias, float* state,
                     long long state_stride, const int* __restrict__ cu_q, const int* __restrict__ seq_rows,
                     T* __restrict__ out, int width) {
    // (A, B) of this CTA's 64 channels: per warp, of the whole CTA (read by the cluster), and of every CTA of the
    // cluster.  The first two exist twice: a turn's values may still be read while the next turn's are written.
    __shared__ float2 warp_ab[2][kWarps][kChannels];
    __shared__ float2 cta_ab[2][kChannels];
    __shared__ float2 all_ab[kMaxCluster][kChannels];
    cg::cluster_group cluster = cg::this_cluster();
    const int ctas = gridDim.x, rank = blockIdx.x;               // the cluster spans the grid's x
    const int entry = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.y * kChannels + 2 * lane;
    const bool live = c < width;
    const int cc = live ? c : 0;                                 // lanes without channels read channel 0 and write nothing
    const int tok0 = cu_q[entry];
    const int q_len = cu_q[entry + 1] - tok0;
    float* srow = state + (size_t)seq_rows[entry] * state_stride;
    const float2 bz = read2<false>(bias, cc, width), bu = read2<false>(bias + width, cc, width);
    float2 carry = read2<false>(srow, cc, width);                // the state before this turn's tokens (all warps agree)

    int buf = 0;
    for (int base = 0; base < q_len; base += ctas * kTile, buf ^= 1) {
        const int t0 = base + rank * kTile + warp * kTokens;
        const int n = min(max(q_len - t0, 0), kTokens);
        const T* row = proj + (size_t)(tok0 + t0) * pitch;
        float2 keep[kTokens], add[kTokens];
        typename Stored<T>::type gates[kTokens];
        float2 A = make_float2(1.f, 1.f), B = make_float2(0.f, 0.f);
        if (n > 0) {
            // No branch between the tokens (their chains of special functions overlap): a token beyond the last is
            // the last one read again, and changes nothing.
#pragma unroll
            for (int i = 0; i < kTokens; ++i) {
                const T* r = row + (size_t)min(i, n - 1) * pitch;
                keep[i] = read2<PAIR>(r, cc, width);
                add[i] = read2<PAIR>(r + width, cc, width);
                gates[i] = read_stored<PAIR>(r + 2 * width, cc, width);
            }
#pragma unroll
            for (int i = 0; i < kTokens; ++i) {
                const float2 z = keep[i], u = add[i];
                cell<T>(z.x + bz.x, u.x + bu.x, keep[i].x, add[i].x);
                cell<T>(z.y + bz.y, u.y + bu.y, keep[i].y, add[i].y);
                if (i >= n) { keep[i] = make_float2(1.f, 1.f); add[i] = make_float2(0.f, 0.f); }
            }
#pragma unroll
            for (int i = 0; i < kTokens; ++i) {
                A.x *= keep[i].x; B.x = keep[i].x * B.x + add[i].x;
                A.y *= keep[i].y; B.y = keep[i].y * B.y + add[i].y;
            }
        }
        warp_ab[buf][warp][2 * lane] = make_float2(A.x, B.x);
        warp_ab[buf][warp][2 * lane + 1] = make_float2(A.y, B.y);
        __syncthreads();
        if (threadIdx.x < kChannels) {
            float2 f = warp_ab[buf][0][threadIdx.x];
#pragma unroll
            for (int w = 1; w < kWarps; ++w) {
                const float2 x = warp_ab[buf][w][threadIdx.x];
                f = make_float2(f.x * x.x, x.x * f.y + x.y);
            }
            cta_ab[buf][threadIdx.x] = f;
        }
        cluster.sync();
        if (warp < ctas) {                                       // a warp per CTA of the cluster brings that CTA's pairs over
            const float2* far = cluster.map_shared_rank(&cta_ab[buf][0], warp);
            all_ab[warp][2 * lane] = far[2 * lane];
            all_ab[warp][2 * lane + 1] = far[2 * lane + 1];
        }
        __syncthreads();
        float2 s = carry;
        for (int r = 0; r < ctas; ++r) {
            if (r == rank) s = carry;
            const float2 a = all_ab[r][2 * lane], b = all_ab[r][2 * lane + 1];
            carry.x = a.x * carry.x + a.y;
            carry.y = b.x * carry.y + b.y;
        }
        for (int w = 0; w < warp; ++w) {
            const float2 a = warp_ab[buf][w][2 * lane], b = warp_ab[buf][w][2 * lane + 1];
            s.x = a.x * s.x + a.y;
            s.y = b.x * s.y + b.y;
        }
        if (n > 0) {
            T* dst = out + (size_t)(tok0 + t0) * width;
            const int last = live ? n : 0;
#pragma unroll
            for (int i = 0; i < kTokens; ++i) {
                s.x = keep[i].x * s.x + add[i].x;
                s.y = keep[i].y * s.y + add[i].y;
                const float2 g = unpack(gates[i]);
                const float2 y = make_float2(s.x * silu<T>(g.x), s.y * silu<T>(g.y));
                if (i < last) write2<PAIR>(dst + (size_t)i * width, cc, width, y);
            }
        }
    }
    // The state goes back after an exchange: every CTA has read the old one.  No CTA leaves while another may still
    // read its pairs.
    if (q_len > 0 && rank == 0 && warp == 0 && live) write2<false>(srow, cc, width, carry);
    cluster.sync();
}

template <typename T>
static bool pairs(const T* proj, int pitch, const T* out, int width) {
    const uintptr_t mask = 2 * sizeof(T) - 1;
    return (width & 1) == 0 && (pitch & 1) == 0 && (((uintptr_t)proj | (uintptr_t)out) & mask) == 0;
}

}  // namespace gru
}  // namespace se

// proj [tokens, 3 * width] (rows `pitch` apart) and out [tokens, width]: the activation type; bias [2 * width] = b_z, b_u
// and state: 32-bit; cu_q [entries + 1], seq_rows [entries].
extern "C" int se_min_gru_scan(const void* proj, int pitch, const float* bias, float* state, long long state_stride,
                               const int* cu_q, const int* seq_rows, void* out, int entries, int width, int dtype,
                               cudaStream_t stream) {
    if (entries <= 0) return 0;
    if (width <= 0 || entries > 65535) return SE_ERR_UNSUPPORTED;
    if (pitch < 3 * width || state_stride < width) return SE_ERR_ARGUMENT;
    const int threads = 128;
    dim3 grid(se::ceil_div(se::ceil_div(width, 2), threads), entries);
    SE_DISPATCH_DTYPE(dtype, T, {
        auto kernel = se::gru::pairs((const T*)proj, pitch, (const T*)out, width) ? se::gru::min_gru_scan_kernel<T, true>
                                                                                 : se::gru::min_gru_scan_kernel<T, false>;
        cudaError_t e = SE_LAUNCH_DEPENDENT("gru", kernel, grid, dim3(threads), 0, stream, (const T*)proj, pitch, bias, state,
                                             state_stride, cu_q, seq_rows, (T*)out, width);
        if (e != cudaSuccess) return (int)e;
    });
    SE_LAUNCH_CHECK();
}

// The same for steps with prompt portions; `ctas` (1, 2, 4 or 8) CTAs share an entry's tokens.
extern "C" int se_min_gru_chunk(const void* proj, int pitch, const float* bias, float* state, long long state_stride,
                                const int* cu_q, const int* seq_rows, void* out, int entries, int width, int ctas, int dtype,
                                cudaStream_t stream) {
    if (entries <= 0) return 0;
    const int blocks = se::ceil_div(width, se::gru::kChannels);
    if (width <= 0 || entries > 65535 || blocks > 65535) return SE_ERR_UNSUPPORTED;
    if (pitch < 3 * width || state_stride < width || !(ctas == 1 || ctas == 2 || ctas == 4 || ctas == 8)) return SE_ERR_ARGUMENT;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(ctas, blocks, entries);
    cfg.blockDim = dim3(32 * se::gru::kWarps);
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = ctas;
    attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    SE_DISPATCH_DTYPE(dtype, T, {
        auto kernel = se::gru::pairs((const T*)proj, pitch, (const T*)out, width) ? se::gru::min_gru_chunk_kernel<T, true>
                                                                                 : se::gru::min_gru_chunk_kernel<T, false>;
        cudaError_t e = cudaLaunchKernelEx(&cfg, kernel, (const T*)proj, pitch, bias, state, state_stride, cu_q, seq_rows,
                                           (T*)out, width);
        if (e != cudaSuccess) return (int)e;
    });
    SE_LAUNCH_CHECK();
}

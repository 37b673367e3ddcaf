// Query/key preparation in its general form, for attention variants the rotary kernel of
// qk_prep.cu does not cover: a value head size of its own, a query temperature that grows with
// the position, layers that bring queries only (they attend over another layer's keys), and
// values blended with those of an earlier layer.
//
//   q_out[t] = rot(q * inv_rms(q) * q_w, pos) * temp(pos)      (statistics over the whole projection)
//   K page   = rot(k * inv_rms(k) * k_w, pos)
//   V page   = v, or (1 - mix) * v + mix * v_first              (v_first: the same token's values elsewhere)
//   temp(p)  = 1 + coef * ln(floor((p + 1) / every) + 1)        (coef = 0: none)
//   rot      : on the first `rotary_dim` dims of every head, dim i paired with dim i + rotary_dim/2 (or, `interleaved`,
//              dim 2i with dim 2i + 1), (u, v) -> (u cos a - v sin a, v cos a + u sin a), a = pos * inv_freq[i], cos and
//              sin multiplied by `rope_scale`  (rotary_dim = 0: none)
//
// Options: `bias` (32-bit, [q | k | v] like the projection row) is added to the projection before
// anything else; `per_head` 1 norms every head by its own root mean square, with weights of d elements
// shared by the heads, instead of the whole projection with a weight per column; `per_head` 2 does so for
// queries and keys without weights, and its root mean square is that of the rotated head (a rotation keeps a pair's
// sum of squares, so the squares of the rotated dims are counted rope_scale^2 times and nothing is rotated twice).
//
// Everything is computed in 32-bit and rounded once.  The norm weights are
// optional.  The projection row is [q: hq*d | k: hkv*d | v: hkv*dv] (`has_kv`) or [q] alone.
//
// Cache layout of one cache layer: per page the keys [kv head][slot in page][d], then the values
// [kv head][slot in page][dv]; with dv = d this is the layout of the other attention kernels.
#include "common.cuh"

namespace se {

constexpr int kMaxHalf = 128;       // half of the largest rotated width (head sizes up to 256)

template <typename T>
__global__ void __launch_bounds__(256)
qk_prep_general_kernel(const T* proj, int pitch, const T* __restrict__ q_w, const T* __restrict__ k_w,
                       const float* __restrict__ inv_freq, int rotary_dim, const T* v_first, int v_first_pitch,
                       const float* __restrict__ v_mix,
                       const int* __restrict__ positions, const int* __restrict__ token_seq,
                       const int* __restrict__ seq_rows, const int* __restrict__ table, int table_stride,
                       T* __restrict__ cache, T* __restrict__ q_out, int hq, int hkv, int d, int dv, float eps,
                       float temp_coef, int temp_every, int page_size, int has_kv, int num_pages, int* __restrict__ error,
                       const float* __restrict__ bias, int per_head, int interleaved, float rope_scale) {
    extern __shared__ float inv_head[];      // per_head: the inverse root mean square of every q head, then every k head
    __shared__ float scratch[33];
    grid_dependency_trigger();
    grid_dependency_wait();      // proj is not __restrict__: its loads stay below this line
    const int t = blockIdx.x;
    const int qn = hq * d, kn = hkv * d, vn = hkv * dv;
    const int pos = positions[t];
    int page = 0;
    if (has_kv) {
        page = table[(size_t)seq_rows[token_seq[t]] * table_stride + pos / page_size];
        if (!page_in_pool(page, num_pages, error, SE_CODE_BAD_PAGE_QK_PREP)) has_kv = 0;
    }
    float temp = 1.f;
    if (temp_coef != 0.f && temp_every > 0) temp = 1.f + temp_coef * logf((float)((pos + 1) / temp_every) + 1.f);
    const T* row = proj + (size_t)t * pitch;
    const int half = rotary_dim / 2;
    const T* vf = v_first != nullptr ? v_first + (size_t)t * v_first_pitch : nullptr;
    // Eight elements at a time where sizes and addresses allow it.
    const bool vec = (d & 7) == 0 && (interleaved ? (rotary_dim & 7) == 0 : (half & 7) == 0) && (dv & 7) == 0 && (pitch & 7) == 0 && aligned8(proj) && aligned8(q_out) &&
                     (bias == nullptr || aligned8(bias)) &&
                     (q_w == nullptr || aligned8(q_w)) && (k_w == nullptr || aligned8(k_w)) && (cache == nullptr || aligned8(cache)) &&
                     (vf == nullptr || ((v_first_pitch & 7) == 0 && aligned8(v_first)));
    // element i of a part of the projection row (its bias starts at bias + b0)
    auto raw = [&](const T* part, int b0, int i) { return to_float(part[i]) + (bias != nullptr ? bias[b0 + i] : 0.f); };
    auto raw8 = [&](const T* part, int b0, int i, float* v) {
        load8(part + i, v);
        if (bias != nullptr) {
            float bb[8];
            load8(bias + b0 + i, bb);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] += bb[j];
        }
    };
    auto sum_squares = [&](const T* part, int b0, int n) {
        float ss = 0.f;
        if (vec) {
            for (int i = threadIdx.x * 8; i < n; i += blockDim.x * 8) {
                float v[8];
                raw8(part, b0, i, v);
#pragma unroll
                for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
            }
        } else {
            for (int i = threadIdx.x; i < n; i += blockDim.x) { const float v = raw(part, b0, i); ss += v * v; }
        }
        return block_sum(ss, scratch);
    };
    float inv_q = 1.f, inv_k = 1.f;
    if (per_head) {
        // a warp per head: q heads (if normed), then k heads
        const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
        const int heads = hq + (has_kv ? hkv : 0);
        for (int h = warp; h < heads; h += warps) {
            const bool is_q = h < hq;
            float ss = 0.f;
            const bool normed = per_head == 2 || (is_q ? q_w : k_w) != nullptr;
            if (normed) {
                const T* part = is_q ? row + (size_t)h * d : row + qn + (size_t)(h - hq) * d;
                const int b0 = is_q ? h * d : qn + (h - hq) * d;
                const float rot2 = per_head == 2 ? rope_scale * rope_scale : 1.f;
                for (int i = lane; i < d; i += 32) { const float v = raw(part, b0, i); ss += i < rotary_dim ? rot2 * v * v : v * v; }
                ss = warp_sum(ss);
            }
            if (lane == 0) inv_head[h] = normed ? 1.0f / sqrtf(ss / (float)d + eps) : 1.f;
        }
        __syncthreads();
    } else {
        if (q_w != nullptr) inv_q = 1.0f / sqrtf(sum_squares(row, 0, qn) / (float)qn + eps);
        if (k_w != nullptr && has_kv) inv_k = 1.0f / sqrtf(sum_squares(row + qn, qn, kn) / (float)kn + eps);
    }
    // cos and sin of the token's angles, once for all heads
    __shared__ float cs_t[kMaxHalf], sn_t[kMaxHalf];
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, cs;
        sincosf((float)pos * inv_freq[i], &sn, &cs);
        sn_t[i] = sn * rope_scale;
        cs_t[i] = cs * rope_scale;
    }
    __syncthreads();
    T* kbase = nullptr;
    T* vbase = nullptr;
    if (has_kv) {
        const size_t page_elems = (size_t)hkv * page_size * (d + dv);
        kbase = cache + (size_t)page * page_elems + (size_t)(pos % page_size) * d;
        vbase = cache + (size_t)page * page_elems + (size_t)hkv * page_size * d + (size_t)(pos % page_size) * dv;
    }
    const float mix = v_first != nullptr ? v_mix[0] : 0.f;
    T* qdst = q_out + (size_t)t * qn;

    // The 8-wide path: a work item is a pair of 8-element chunks that rotate into one another (columns c
    // and c + half of a head), or one chunk that passes.
    if (vec) {
        const int pair_items = interleaved ? 0 : half / 8, items = d / 8 - pair_items;          // per head
        auto normed8 = [&](const T* part, int b0, const T* w, float inv, int i, int wi, float* v) {
            raw8(part, b0, i, v);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] *= inv;
            if (w != nullptr) {
                float ww[8];
                load8(w + wi, ww);
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] *= ww[j];
            }
        };
        // heads of the queries, then (with keys) heads of the keys
        const int heads = hq + (has_kv ? hkv : 0);
        for (int it = threadIdx.x; it < heads * items; it += blockDim.x) {
            const int h = it / items, k = it - h * items;
            const bool is_q = h < hq;
            const int hh = is_q ? h : h - hq;
            const T* part = is_q ? row : row + qn;
            const int b0 = is_q ? 0 : qn;
            const T* w = is_q ? q_w : k_w;
            const float inv = per_head ? inv_head[h] : (is_q ? inv_q : inv_k), mul = is_q ? temp : 1.f;
            const int w0 = per_head ? 0 : hh * d;        // where the head's weights start
            T* dst = is_q ? qdst + (size_t)hh * d : kbase + (size_t)hh * page_size * d;
            float a[8];
            if (k < pair_items) {
                const int c = k * 8;
                float b[8], ra[8], rb[8];
                normed8(part, b0, w, inv, hh * d + c, w0 + c, a);
                normed8(part, b0, w, inv, hh * d + c + half, w0 + c + half, b);
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    const float cs = cs_t[c + j], sn = sn_t[c + j];
                    ra[j] = (a[j] * cs - b[j] * sn) * mul;
                    rb[j] = (b[j] * cs + a[j] * sn) * mul;
                }
                store8(dst + c, ra);
                store8(dst + c + half, rb);
            } else {
                const int c = interleaved ? k * 8 : rotary_dim + (k - pair_items) * 8;
                normed8(part, b0, w, inv, hh * d + c, w0 + c, a);
                if (interleaved && c < rotary_dim) {
#pragma unroll
                    for (int j = 0; j < 8; j += 2) {
                        const float cs = cs_t[(c + j) / 2], sn = sn_t[(c + j) / 2], u = a[j], v = a[j + 1];
                        a[j] = u * cs - v * sn;
                        a[j + 1] = v * cs + u * sn;
                    }
                }
#pragma unroll
                for (int j = 0; j < 8; ++j) a[j] *= mul;
                store8(dst + c, a);
            }
        }
        if (!has_kv) return;
        for (int i = threadIdx.x * 8; i < vn; i += blockDim.x * 8) {
            const int h = i / dv, c = i - h * dv;
            if (vf == nullptr && bias == nullptr) {
                *reinterpret_cast<uint4*>(vbase + (size_t)h * page_size * dv + c) = *reinterpret_cast<const uint4*>(row + qn + kn + i);
                if (sizeof(T) == 4)
                    *reinterpret_cast<uint4*>(vbase + (size_t)h * page_size * dv + c + 4) = *reinterpret_cast<const uint4*>(row + qn + kn + i + 4);
            } else {
                float a[8], f[8];
                raw8(row + qn + kn, qn + kn, i, a);
                if (vf != nullptr) {
                    load8(vf + i, f);
#pragma unroll
                    for (int j = 0; j < 8; ++j) a[j] = (1.f - mix) * a[j] + mix * f[j];
                }
                store8(vbase + (size_t)h * page_size * dv + c, a);
            }
        }
        return;
    }

    // element i of a projection part (norm weights w, inverse root mean square inv), normed and rotated
    auto prepared = [&](const T* part, int b0, const T* w, float inv_whole, int h0, int i) {
        const int c = i % d;
        const float inv = per_head ? inv_head[h0 + i / d] : inv_whole;
        float v = raw(part, b0, i) * inv;
        if (w != nullptr) v *= to_float(w[per_head ? c : i]);
        if (c >= rotary_dim) return v;
        const bool first = interleaved ? (c & 1) == 0 : c < half;
        const int step = interleaved ? 1 : half, j = first ? i + step : i - step;
        const int pair = interleaved ? c / 2 : first ? c : c - half;
        float u = raw(part, b0, j) * inv;
        if (w != nullptr) u *= to_float(w[per_head ? j % d : j]);
        const float sn = sn_t[pair], cs = cs_t[pair];
        return first ? v * cs - u * sn : v * cs + u * sn;
    };
    for (int i = threadIdx.x; i < qn; i += blockDim.x)
        qdst[i] = from_float<T>(prepared(row, 0, q_w, inv_q, 0, i) * temp);
    if (!has_kv) return;
    for (int i = threadIdx.x; i < kn; i += blockDim.x) {
        const int h = i / d, c = i - h * d;
        kbase[(size_t)h * page_size * d + c] = from_float<T>(prepared(row + qn, qn, k_w, inv_k, hq, i));
    }
    for (int i = threadIdx.x; i < vn; i += blockDim.x) {
        const int h = i / dv, c = i - h * dv;
        float v = raw(row + qn + kn, qn + kn, i);
        if (vf != nullptr) v = (1.f - mix) * v + mix * to_float(vf[i]);
        vbase[(size_t)h * page_size * dv + c] = from_float<T>(v);
    }
}

// Per-head work and nothing else: biases, per-head norms (NORM 1 with weights, 2 without, 0 none) and a rotation (ROT 1
// split halves, 2 neighbours, 0 none); no temperature and no blending.  Every 16-byte chunk (float32: two) of the step's
// projection rows is a lane's work item.  With norms a head's d / 8 chunks lie in neighbouring lanes of one warp (d / 8 a
// power of two), so its sum of squares is a few shuffles; split halves read the partner's chunk once more.  Cosines
// and sines of the tokens a block meets are worked out once, in shared memory.
constexpr int kPrepItems = 256;      // work items (threads) of a block
__host__ __device__ __forceinline__ int prep_block_tokens(int per_token) { return kPrepItems / per_token + 2; }

template <typename T, int NORM, int ROT>
__global__ void __launch_bounds__(kPrepItems)
qk_prep_heads_kernel(const T* proj, int pitch, const T* __restrict__ q_w, const T* __restrict__ k_w,
                     const float* __restrict__ inv_freq, int rotary_dim, float rope_scale, const float* __restrict__ bias,
                     const int* __restrict__ positions, const int* __restrict__ token_seq, const int* __restrict__ seq_rows,
                     const int* __restrict__ table, int table_stride, T* cache, T* q_out, unsigned items, int hq, int hkv,
                     int d, int dv, float eps, int page_size, int num_pages, int* __restrict__ error) {
    extern __shared__ float2 turns[];            // [tokens of the block][rotary_dim / 2]: (cos, sin) * rope_scale
    grid_dependency_trigger();
    const int lanes = d / 8, qc = hq * lanes, kc = hkv * lanes, per_token = qc + kc + hkv * (dv / 8);
    const unsigned x0 = blockIdx.x * kPrepItems, x = x0 + threadIdx.x;
    const int t_first = (int)(x0 / per_token), half = rotary_dim / 2;
    const int from = (int)(x0 - (unsigned)t_first * per_token);       // the block's first item within its first token
    grid_dependency_wait();
    if (ROT) {
        const int count = (int)min((unsigned)kPrepItems, items - x0);
        const int n = ((from + count - 1) / per_token + 1) * half;
        for (int i = threadIdx.x; i < n; i += kPrepItems) {
            const int t = i / half;
            float sn, cs;
            sincosf((float)positions[t_first + t] * inv_freq[i - t * half], &sn, &cs);
            turns[i] = make_float2(cs * rope_scale, sn * rope_scale);
        }
    }
    const bool live = x < items;
    const int ahead = live ? (from + (int)threadIdx.x) / per_token : 0;
    const int t = t_first + ahead;
    const int c = live ? from + (int)threadIdx.x - ahead * per_token : 0;
    const T* row = proj + (size_t)t * pitch;
    auto load_raw = [&](int chunk, float* v) {
        load8(row + 8 * chunk, v);
        if (bias != nullptr) {
            float b[8];
            load8(bias + 8 * chunk, b);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] += b[j];
        }
    };
    float v[8];
    load_raw(c, v);
    const bool is_q = c < qc, is_v = c >= qc + kc;
    const int head = is_v ? 0 : c / lanes;
    const int in_head = is_v ? 0 : (c - head * lanes) * 8;
    float inv = 1.f;
    if (NORM) {
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
        // a chunk rotates as a whole or not at all (rotary_dim a multiple of 8)
        if (NORM == 2 && ROT && in_head < rotary_dim) ss *= rope_scale * rope_scale;
        for (int o = lanes / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);       // items of values: a sum nobody uses
        inv = 1.0f / sqrtf(ss / (float)d + eps);
    }
    if (ROT) __syncthreads();
    if (!live) return;
    if (!is_v) {
        const T* w = is_q ? q_w : k_w;
        auto weigh = [&](int at, float* a) {
#pragma unroll
            for (int j = 0; j < 8; ++j) a[j] *= inv;
            if (NORM == 1) {
                float wv[8];
                load8(w + at, wv);
#pragma unroll
                for (int j = 0; j < 8; ++j) a[j] *= wv[j];
            }
        };
        if (NORM) weigh(in_head, v);
        if (ROT == 1 && in_head < rotary_dim) {
            const bool first = in_head < half;
            const int other = first ? in_head + half : in_head - half;
            float u[8];
            load_raw(head * lanes + other / 8, u);
            if (NORM) weigh(other, u);
            const float2* cs = turns + (size_t)(t - t_first) * half + (first ? in_head : other);
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = first ? v[j] * cs[j].x - u[j] * cs[j].y : v[j] * cs[j].x + u[j] * cs[j].y;
        }
        if (ROT == 2 && in_head < rotary_dim) {
            const float2* cs = turns + (size_t)(t - t_first) * half + in_head / 2;
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                const float a = v[j], b = v[j + 1];
                v[j] = a * cs[j / 2].x - b * cs[j / 2].y;
                v[j + 1] = b * cs[j / 2].x + a * cs[j / 2].y;
            }
        }
        if (is_q) {
            store8(q_out + ((size_t)t * qc + c) * 8, v);
            return;
        }
    }
    const int pos = positions[t];
    const int page = table[(size_t)seq_rows[token_seq[t]] * table_stride + pos / page_size];
    if (!page_in_pool(page, num_pages, error, SE_CODE_BAD_PAGE_QK_PREP)) return;
    const int slot = pos % page_size;
    T* base = cache + (size_t)page * hkv * page_size * (d + dv);
    if (!is_v) {
        store8(base + ((size_t)(head - hq) * page_size + slot) * d + in_head, v);
    } else {
        const int i = (c - qc - kc) * 8, h = i / dv;
        store8(base + (size_t)hkv * page_size * d + ((size_t)h * page_size + slot) * dv + (i - h * dv), v);
    }
}

}  // namespace se

extern "C" int se_qk_prep_general(const void* proj, int pitch, const void* q_w, const void* k_w, const float* inv_freq,
                                  int rotary_dim, const void* v_first, int v_first_pitch, const float* v_mix,
                                  const int* positions,
                                  const int* token_seq, const int* seq_rows, const int* table, int table_stride,
                                  void* cache, void* q_out, int tokens, int hq, int hkv, int d, int dv, float eps,
                                  float temp_coef, int temp_every, int page_size, int has_kv, int num_pages, int* error,
                                  const float* bias, int per_head, int interleaved, float rope_scale, int dtype,
                                  cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (hq <= 0 || d <= 0 || (has_kv && (hkv <= 0 || dv <= 0 || page_size <= 0))) return SE_ERR_ARGUMENT;
    if (pitch < hq * d + (has_kv ? hkv * (d + dv) : 0)) return SE_ERR_ARGUMENT;
    if (rotary_dim < 0 || rotary_dim > d || (rotary_dim & 1) || (rotary_dim > 0 && inv_freq == nullptr)) return SE_ERR_ARGUMENT;
    if (rotary_dim > 2 * se::kMaxHalf) return SE_ERR_UNSUPPORTED;
    if (rotary_dim == 0) rope_scale = 1.f;
    if (v_first != nullptr && (v_mix == nullptr || !has_kv || v_first_pitch < hkv * dv)) return SE_ERR_ARGUMENT;
    // per-head work alone, in chunks of 8 elements
    const size_t esize = dtype == SE_DTYPE_F32 ? 4 : 2;
    auto aligned = [](const void* p) { return p == nullptr || (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const int lanes = d / 8, per_token = hkv > 0 ? (hq + hkv) * lanes + hkv * (dv / 8) : 0;
    const bool normed = per_head != 0, lanes_fit = lanes >= 1 && lanes <= 32 && (lanes & (lanes - 1)) == 0 && (hkv * (dv / 8)) % lanes == 0;
    if (has_kv && (normed ? lanes_fit && (per_head == 2 || (q_w != nullptr && k_w != nullptr)) : q_w == nullptr && k_w == nullptr) &&
        (normed || rotary_dim > 0 || bias != nullptr) && (temp_coef == 0.f || temp_every <= 0) && v_first == nullptr && (d & 7) == 0 && (dv & 7) == 0 &&
        (interleaved ? (rotary_dim & 7) == 0 : (rotary_dim & 15) == 0) && (pitch * esize) % 16 == 0 && aligned(proj) &&
        aligned(q_out) && aligned(cache) && aligned(q_w) && aligned(k_w) && aligned(bias)) {
        const long long items = (long long)tokens * per_token;
        const long long blocks = (items + se::kPrepItems - 1) / se::kPrepItems;
        if (items > 0x7fffff00LL) return SE_ERR_UNSUPPORTED;
        const size_t turns = rotary_dim > 0 ? (size_t)se::prep_block_tokens(per_token) * (rotary_dim / 2) * sizeof(float2) : 0;
        const int norm = per_head, rot = rotary_dim == 0 ? 0 : interleaved ? 2 : 1;
#define SE_PREP_CASE(N, R)                                                                                                  \
    if (norm == N && rot == R)                                                                                              \
        e = SE_LAUNCH_DEPENDENT("qk", (se::qk_prep_heads_kernel<T, N, R>), dim3((unsigned)blocks), dim3(se::kPrepItems), turns, stream, \
                                 (const T*)proj, pitch, (const T*)q_w, (const T*)k_w, inv_freq, rotary_dim, rope_scale, bias, \
                                 positions, token_seq, seq_rows, table, table_stride, (T*)cache, (T*)q_out, (unsigned)items, hq, hkv, d, \
                                 dv, eps, page_size, num_pages, error);
        SE_DISPATCH_DTYPE(dtype, T, {
            cudaError_t e = cudaErrorInvalidValue;
            SE_PREP_CASE(0, 0) SE_PREP_CASE(0, 1) SE_PREP_CASE(0, 2) SE_PREP_CASE(1, 0) SE_PREP_CASE(1, 1) SE_PREP_CASE(1, 2)
            SE_PREP_CASE(2, 0) SE_PREP_CASE(2, 1) SE_PREP_CASE(2, 2)
            if (e != cudaSuccess) return (int)e;
        });
#undef SE_PREP_CASE
        SE_LAUNCH_CHECK();
    }
    const size_t smem = per_head ? (size_t)(hq + (has_kv ? hkv : 0)) * sizeof(float) : 0;
    if (smem > 40 * 1024) return SE_ERR_UNSUPPORTED;
    SE_DISPATCH_DTYPE(dtype, T, {
        cudaError_t e = SE_LAUNCH_DEPENDENT("qk", se::qk_prep_general_kernel<T>, dim3(tokens), dim3(256), smem, stream,
                                             (const T*)proj, pitch, (const T*)q_w, (const T*)k_w, inv_freq, rotary_dim, (const T*)v_first,
                                             v_first_pitch, v_mix, positions, token_seq, seq_rows,
                                             table, table_stride, (T*)cache, (T*)q_out, hq, hkv, d, dv, eps, temp_coef, temp_every,
                                             page_size, has_kv, num_pages, error, bias, per_head, interleaved, rope_scale);
        if (e != cudaSuccess) return (int)e;
    });
    SE_LAUNCH_CHECK();
}

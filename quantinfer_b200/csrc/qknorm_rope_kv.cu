// Per-head RMSNorm of q and k, rotary position encoding, and the write of k
// and v into the request's cache pages, in one pass over the fused qkv rows.
//
// Order, as the reference runs it (crates/quantinfer-runtime/src/qwen3/mod.rs:182-183,
// batch.rs:30-55): q and k are normalised over head_dim with one gain vector
// shared by all heads (backends/cpu/src/backend.rs:195-203), then rotated
// (half-split pairs (p, p + rot/2); backends/cpu/src/backend.rs:270-275), then k
// (rotated) and v (raw) are appended to the cache (cache.rs:94-127).
// The pairing rule is a parameter: `interleaved` rotates adjacent elements (2p, 2p + 1)
// with the angle of pair p instead, the order the reference's converter produces for
// architectures it stores that way (crates/quantinfer-format/src/gguf/layout.rs:52-55).
// A position beyond the rotation table sets a status bit and uses the table's last row.
// Norm sums, angles and the rotation are 32-bit. cos/sin come from a table
// [max_positions, rot/2] built once by rope_table below from 32-bit inverse
// frequencies (attention.rs:29-32: angle = position * theta^(-2p/d)).
//
// Cache pages of one layer: [num_pages, kv_heads, page_size, head_dim]; the
// token at position p of request r lies in page table[r, p / page_size] at row
// p % page_size.
#include "common.cuh"
#include "vec8.cuh"

namespace {

constexpr int kWarpsPerBlock = 4;
constexpr int kMaxHeadDim = 512;

template <typename T>
__global__ void qk_norm_rope_kv_kernel(
    const T* __restrict__ qkv, T* __restrict__ q_out, const float* __restrict__ q_gain,
    const float* __restrict__ k_gain, float eps, const float* __restrict__ cos_t,
    const float* __restrict__ sin_t, int rot, int interleaved, int table_positions, const int* __restrict__ positions,
    const int* __restrict__ token_req, const int* __restrict__ block_table, int max_blocks,
    int page_size, int num_pages, T* __restrict__ k_pages, T* __restrict__ v_pages, int nq, int nkv,
    int d, int* __restrict__ status) {
    qi::pdl_enter();
    const int t = blockIdx.x;
    const int head = blockIdx.y * kWarpsPerBlock + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    const int total_heads = nq + 2 * nkv;
    if (head >= total_heads) return;
    const int row_width = total_heads * d;
    const T* src = qkv + (size_t)t * row_width + (size_t)head * d;
    const int pos = positions[t];
    if (pos < 0) {
        if (lane == 0 && status) atomicOr(status, qi::kStatusBadRange);
        return;
    }
    int table_row = pos;
    if (cos_t && pos >= table_positions) {
        if (lane == 0 && status) atomicOr(status, qi::kStatusBadRange);
        table_row = table_positions - 1;
    }

    // Destination row.
    T* dst = nullptr;
    const bool is_q = head < nq;
    const bool is_k = !is_q && head < nq + nkv;
    if (is_q) {
        dst = q_out + (size_t)t * nq * d + (size_t)head * d;
    } else {
        if (k_pages == nullptr) return;  // a layer that reads another layer's cache writes none
        const int hk = is_k ? head - nq : head - nq - nkv;
        const int r = token_req[t];
        const int page = block_table[(size_t)r * max_blocks + pos / page_size];
        if (page < 0 || page >= num_pages) {
            if (lane == 0 && status) atomicOr(status, qi::kStatusBadPage);
            return;
        }
        T* base = is_k ? k_pages : v_pages;
        dst = base + (((size_t)page * nkv + hk) * page_size + (pos % page_size)) * (size_t)d;
    }

    if (!is_q && !is_k) {  // v: raw copy
        for (int i = lane; i < d; i += 32) dst[i] = src[i];
        return;
    }

    const float* gain = is_q ? q_gain : k_gain;
    float inv = 1.f;
    if (gain) {
        float ss = 0.f;
        for (int i = lane; i < d; i += 32) {
            const float v = qi::to_f32<T>(src[i]);
            ss += v * v;
        }
        ss = qi::warp_sum(ss);
        inv = 1.0f / sqrtf(ss / (float)d + eps);
    }
    const int half = rot / 2;
    // Rotated pairs.
    for (int p = lane; p < half; p += 32) {
        const int ia = interleaved ? 2 * p : p, ib = interleaved ? 2 * p + 1 : p + half;
        float a = qi::to_f32<T>(src[ia]);
        float b = qi::to_f32<T>(src[ib]);
        if (gain) {
            a = a * inv * gain[ia];
            b = b * inv * gain[ib];  // stays 32-bit until after the rotation
        }
        float c = 1.f, s = 0.f;
        if (cos_t) {
            c = cos_t[(size_t)table_row * half + p];
            s = sin_t[(size_t)table_row * half + p];
        }
        dst[ia] = qi::from_f32<T>(a * c - b * s);
        dst[ib] = qi::from_f32<T>(a * s + b * c);
    }
    // Dimensions beyond the rotary part pass through (normalised).
    for (int i = rot + lane; i < d; i += 32) {
        float a = qi::to_f32<T>(src[i]);
        if (gain) a = a * inv * gain[i];
        dst[i] = qi::from_f32<T>(a);
    }
}

// Two adjacent elements per access (head_dim a multiple of 4, rotation over the whole head).
template <typename T> struct Pair;
template <> struct Pair<float> {
    static __device__ __forceinline__ float2 load(const float* p) { return *reinterpret_cast<const float2*>(p); }
    static __device__ __forceinline__ void store(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
};
template <> struct Pair<qi::bf16> {
    static __device__ __forceinline__ float2 load(const qi::bf16* p) {
        return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    }
    static __device__ __forceinline__ void store(qi::bf16* p, float a, float b) {
        *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
    }
};

// Sum over the K splits of a product's 32-bit partial sums (one split: the value itself).
template <typename TIn>
__device__ __forceinline__ float2 load_pair(const TIn* p, int splits, size_t stride) {
    float2 v = Pair<TIn>::load(p);
#pragma unroll 4
    for (int k = 1; k < splits; ++k) {
        const float2 w = Pair<TIn>::load(p + k * stride);
        v.x += w.x;
        v.y += w.y;
    }
    return v;
}

// TIn = T: qkv is the projection's output. TIn = float with splits > 1: qkv holds the
// projection's K-split partial sums [splits, n, width], added here in split order.
template <typename TIn, typename T>
__global__ void qk_norm_rope_kv_vec_kernel(
    const TIn* __restrict__ qkv, int splits, size_t split_stride, T* __restrict__ q_out, const float* __restrict__ q_gain,
    const float* __restrict__ k_gain, float eps, const float* __restrict__ cos_t,
    const float* __restrict__ sin_t, int table_positions, const int* __restrict__ positions,
    const int* __restrict__ token_req, const int* __restrict__ block_table, int max_blocks,
    int page_size, int num_pages, T* __restrict__ k_pages, T* __restrict__ v_pages, int nq, int nkv,
    int d, int* __restrict__ status) {
    qi::pdl_enter();
    const int t = blockIdx.x;
    const int head = blockIdx.y * kWarpsPerBlock + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    const int total_heads = nq + 2 * nkv;
    if (head >= total_heads) return;
    const TIn* src = qkv + (size_t)t * total_heads * d + (size_t)head * d;
    const int pos = positions[t];
    if (pos < 0) {
        if (lane == 0 && status) atomicOr(status, qi::kStatusBadRange);
        return;
    }
    int table_row = pos;
    if (cos_t && pos >= table_positions) {
        if (lane == 0 && status) atomicOr(status, qi::kStatusBadRange);
        table_row = table_positions - 1;
    }
    const bool is_q = head < nq;
    const bool is_k = !is_q && head < nq + nkv;
    T* dst;
    if (is_q) {
        dst = q_out + (size_t)t * nq * d + (size_t)head * d;
    } else {
        if (k_pages == nullptr) return;
        const int hk = is_k ? head - nq : head - nq - nkv;
        const int page = block_table[(size_t)token_req[t] * max_blocks + pos / page_size];
        if (page < 0 || page >= num_pages) {
            if (lane == 0 && status) atomicOr(status, qi::kStatusBadPage);
            return;
        }
        dst = (is_k ? k_pages : v_pages) + (((size_t)page * nkv + hk) * page_size + (pos % page_size)) * (size_t)d;
    }
    if (!is_q && !is_k) {
        for (int i = 2 * lane; i < d; i += 64) {
            const float2 v = load_pair<TIn>(src + i, splits, split_stride);
            Pair<T>::store(dst + i, v.x, v.y);
        }
        return;
    }
    const int half = d / 2;
    const float* gain = is_q ? q_gain : k_gain;
    float inv = 1.f;
    if (gain) {
        float ss = 0.f;
        for (int i = 2 * lane; i < d; i += 64) {
            const float2 v = load_pair<TIn>(src + i, splits, split_stride);
            ss += v.x * v.x + v.y * v.y;
        }
        ss = qi::warp_sum(ss);
        inv = 1.0f / sqrtf(ss / (float)d + eps);
    }
    for (int p = 2 * lane; p < half; p += 64) {
        float2 a = load_pair<TIn>(src + p, splits, split_stride), b = load_pair<TIn>(src + p + half, splits, split_stride);
        if (gain) {
            const float2 ga = *reinterpret_cast<const float2*>(gain + p), gb = *reinterpret_cast<const float2*>(gain + p + half);
            a.x = a.x * inv * ga.x; a.y = a.y * inv * ga.y;
            b.x = b.x * inv * gb.x; b.y = b.y * inv * gb.y;
        }
        float2 c = make_float2(1.f, 1.f), sn = make_float2(0.f, 0.f);
        if (cos_t) {
            c = *reinterpret_cast<const float2*>(cos_t + (size_t)table_row * half + p);
            sn = *reinterpret_cast<const float2*>(sin_t + (size_t)table_row * half + p);
        }
        Pair<T>::store(dst + p, a.x * c.x - b.x * sn.x, a.y * c.y - b.y * sn.y);
        Pair<T>::store(dst + p + half, a.x * sn.x + b.x * c.x, a.y * sn.y + b.y * c.y);
    }
}

__global__ void rope_table_kernel(const float* __restrict__ inv_freq, float* __restrict__ cos_t,
                                  float* __restrict__ sin_t, int max_pos, int half) {
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (size_t)max_pos * half) return;
    const int pos = (int)(idx / half), p = (int)(idx % half);
    const float angle = (float)pos * inv_freq[p];
    cos_t[idx] = cosf(angle);
    sin_t[idx] = sinf(angle);
}

}  // namespace

extern "C" int qi_rope_table(const float* inv_freq, float* cos_t, float* sin_t, int max_pos,
                             int half, cudaStream_t stream) {
    QI_REQUIRE(max_pos > 0 && half > 0, "rope_table: bad sizes max_pos=%d half=%d", max_pos, half);
    const size_t n = (size_t)max_pos * half;
    rope_table_kernel<<<(unsigned)((n + 255) / 256), 256, 0, stream>>>(inv_freq, cos_t, sin_t, max_pos,
                                                                      half);
    return qi::check_launch("rope_table");
}

// q_gain/k_gain null: no norm. cos_t null: no rotation. k_pages null: no cache write.
// interleaved: pairs (2p, 2p + 1) instead of (p, p + rot/2).
// qkv_splits > 1: `qkv` holds float32 partial sums [qkv_splits, n_tokens, width] of the projection.
extern "C" int qi_qk_norm_rope_kv(const void* qkv, int qkv_splits, void* q_out, int dtype, const float* q_gain,
                                  const float* k_gain, float eps, const float* cos_t,
                                  const float* sin_t, int rot, int interleaved, int table_positions,
                                  const int* positions, const int* token_req,
                                  const int* block_table, int max_blocks, int page_size,
                                  int num_pages, void* k_pages, void* v_pages, int n_tokens, int nq,
                                  int nkv, int d, int* status, cudaStream_t stream) {
    QI_REQUIRE(n_tokens >= 0 && nq > 0 && nkv > 0 && d > 0, "qk_norm_rope_kv: bad sizes");
    QI_REQUIRE(d <= kMaxHeadDim, "qk_norm_rope_kv: head_dim %d is above the limit %d", d, kMaxHeadDim);
    QI_REQUIRE(rot >= 0 && rot <= d && rot % 2 == 0, "qk_norm_rope_kv: rotary size %d must be even and <= head_dim %d", rot, d);
    QI_REQUIRE(!cos_t || (sin_t && table_positions > 0), "qk_norm_rope_kv: incomplete rotation table");
    QI_REQUIRE((k_pages == nullptr) == (v_pages == nullptr), "qk_norm_rope_kv: k and v pages must come together");
    QI_REQUIRE(!k_pages || (page_size > 0 && max_blocks > 0 && num_pages > 0 && block_table && token_req),
               "qk_norm_rope_kv: incomplete page arguments");
    if (n_tokens == 0) return 0;
    const int heads = nq + 2 * nkv;
    dim3 grid(n_tokens, (heads + kWarpsPerBlock - 1) / kWarpsPerBlock);
    QI_REQUIRE(grid.y <= 65535, "qk_norm_rope_kv: too many heads");
    if (!cos_t) rot = 0;
    QI_REQUIRE(qkv_splits >= 1, "qk_norm_rope_kv: qkv_splits must be >= 1");
    const bool vec = d % 4 == 0 && (rot == d || rot == 0) && (!interleaved || rot == 0) && ((uintptr_t)qkv & 7) == 0 && ((uintptr_t)q_out & 7) == 0 &&
                     ((uintptr_t)k_pages & 7) == 0 && ((uintptr_t)v_pages & 7) == 0;
    if (qkv_splits > 1) {
        QI_REQUIRE(vec, "qk_norm_rope_kv: partial sums as input need head_dim %% 4 == 0 and a half-split rotation over the whole head");
        const size_t stride = (size_t)n_tokens * heads * d;
        QI_DISPATCH_DTYPE(dtype, T, {
            qi::launch(qk_norm_rope_kv_vec_kernel<float, T>, grid, dim3(kWarpsPerBlock * 32), 0, stream,
                (const float*)qkv, qkv_splits, stride, (T*)q_out, q_gain, k_gain, eps, cos_t, sin_t, table_positions, positions, token_req,
                block_table, max_blocks, page_size, num_pages, (T*)k_pages, (T*)v_pages, nq, nkv, d, status);
        });
        return qi::check_launch("qk_norm_rope_kv");
    }
    if (vec) {
        QI_DISPATCH_DTYPE(dtype, T, {
            qi::launch(qk_norm_rope_kv_vec_kernel<T, T>, grid, dim3(kWarpsPerBlock * 32), 0, stream,
                (const T*)qkv, 1, (size_t)0, (T*)q_out, q_gain, k_gain, eps, cos_t, sin_t, table_positions, positions, token_req,
                block_table, max_blocks, page_size, num_pages, (T*)k_pages, (T*)v_pages, nq, nkv, d, status);
        });
        return qi::check_launch("qk_norm_rope_kv");
    }
    QI_DISPATCH_DTYPE(dtype, T, {
        qi::launch(qk_norm_rope_kv_kernel<T>, grid, dim3(kWarpsPerBlock * 32), 0, stream,
            (const T*)qkv, (T*)q_out, q_gain, k_gain, eps, cos_t, sin_t, rot, interleaved, table_positions, positions, token_req,
            block_table, max_blocks, page_size, num_pages, (T*)k_pages, (T*)v_pages, nq, nkv, d,
            status);
    });
    return qi::check_launch("qk_norm_rope_kv");
}

// ---- biases, rotation by angles computed where they are used, and the cache write ----------------------
//
// For designs whose projections have biases, whose values may have another size than their keys, and
// which set no limit on positions (so there is no table): a row of `proj` holds q (nq heads of d), k (nkv
// heads of d) and v (nkv heads of dv) side by side, possibly followed by more columns (`ld` elements a
// row). The bias (32-bit, q | k | v, may be null) is added, the first `rot` coordinates of every q and k
// head turn by angle = position * inv_freq[pair] (32-bit product, sincosf), pairs (i, i + rot / 2) or, when
// `interleaved`, (2i, 2i + 1); q goes to q_out [n, nq d], k and v into the request's pages
// (k_pages [pages, nkv, page_size, d], v_pages [pages, nkv, page_size, dv]; null: nothing is written).
// Options for designs that ask for them: one RMS norm over the whole of q and one over the whole of k (all heads
// at once, gain per coordinate) before the rotation, or one over every head by itself (`head_norm`; a gain of d numbers
// that the heads share); values that are the keys as projected (no v in the row); a factor on q that grows with the
// position, 1 + temp_coef ln(floor((p + 1) / temp_every) + 1); and values mixed with another layer's values of the same
// token (`v_first`, rows `ldv` elements apart): v <- (1 - v_share) v + v_share v_first, in 32-bit.
namespace {

__device__ __forceinline__ float query_factor(int pos, float temp_coef, int temp_every) {
    return temp_every > 0 ? fmaf(temp_coef, logf((float)((pos + 1) / temp_every + 1)), 1.f) : 1.f;
}

template <typename T>
__global__ void __launch_bounds__(256)
bias_rope_kv_kernel(const T* __restrict__ proj, long long ld, const float* __restrict__ bias, T* __restrict__ q_out,
                    const float* __restrict__ inv_freq, int rot, int interleaved, const int* __restrict__ positions,
                    const int* __restrict__ token_req, const int* __restrict__ block_table, int max_blocks, int page_size,
                    int num_pages, T* __restrict__ k_pages, T* __restrict__ v_pages, int nq, int nkv, int d, int dv,
                    const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps, int head_norm, int v_from_k,
                    float temp_coef, int temp_every, const T* __restrict__ v_first, long long ldv, float v_share,
                    int* __restrict__ status) {
    __shared__ float scratch[32];
    extern __shared__ float head_inv[];         // [nq + nkv] with norms of every head by itself
    qi::pdl_wait();
    const int t = blockIdx.x;
    const int pos = positions[t];
    if (pos < 0) {
        if (threadIdx.x == 0 && status) atomicOr(status, qi::kStatusBadRange);
        return;
    }
    const T* row = proj + (size_t)t * ld;
    const int qk = (nq + nkv) * d, total = v_from_k ? qk : qk + nkv * dv;
    // one RMS norm over all of q and one over all of k (before the rotation), when their gains are given
    float q_inv = 1.f, k_inv = 1.f;
    if (q_gain && head_norm) {
        const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
        for (int hd = warp; hd < nq + nkv; hd += blockDim.x >> 5) {
            float sq = 0.f;
            for (int i = lane; i < d; i += 32) {
                const float x = qi::to_f32<T>(row[hd * d + i]) + (bias ? bias[hd * d + i] : 0.f);
                sq = fmaf(x, x, sq);
            }
            sq = qi::warp_sum(sq);
            if (lane == 0) head_inv[hd] = 1.0f / sqrtf(sq / (float)d + eps);
        }
        __syncthreads();
    } else if (q_gain) {
        float sq = 0.f, sk = 0.f;
        for (int e = threadIdx.x; e < qk; e += blockDim.x) {
            const float x = qi::to_f32<T>(row[e]) + (bias ? bias[e] : 0.f);
            if (e < nq * d) sq = fmaf(x, x, sq); else sk = fmaf(x, x, sk);
        }
        q_inv = 1.0f / sqrtf(qi::block_sum(sq, scratch) / (float)(nq * d) + eps);
        k_inv = 1.0f / sqrtf(qi::block_sum(sk, scratch) / (float)(nkv * d) + eps);
    }
    auto normed = [&](int e) {
        float x = qi::to_f32<T>(row[e]) + (bias ? bias[e] : 0.f);
        if (q_gain && head_norm) x = x * head_inv[e / d] * (e < nq * d ? q_gain : k_gain)[e % d];
        else if (q_gain) x = e < nq * d ? x * q_inv * q_gain[e] : x * k_inv * k_gain[e - nq * d];
        return x;
    };
    T* krow = nullptr;
    T* vrow = nullptr;
    if (k_pages) {
        const int page = block_table[(size_t)token_req[t] * max_blocks + pos / page_size];
        if (page < 0 || page >= num_pages) {
            if (threadIdx.x == 0 && status) atomicOr(status, qi::kStatusBadPage);
        } else {
            krow = k_pages + ((size_t)page * nkv * page_size + (pos % page_size)) * (size_t)d;
            vrow = v_pages + ((size_t)page * nkv * page_size + (pos % page_size)) * (size_t)dv;
        }
    }
    const int half = rot / 2;
    const float q_factor = query_factor(pos, temp_coef, temp_every);
    for (int e = threadIdx.x; e < total; e += blockDim.x) {
        if (e >= qk) {   // a value: bias, and another layer's value mixed in
            const int hv = (e - qk) / dv, i = (e - qk) % dv;
            float v = qi::to_f32<T>(row[e]) + (bias ? bias[e] : 0.f);
            if (v_first) v = (1.f - v_share) * v + v_share * qi::to_f32<T>(v_first[(size_t)t * ldv + (e - qk)]);
            if (vrow) vrow[(size_t)hv * page_size * dv + i] = qi::from_f32<T>(v);
            continue;
        }
        const int head = e / d, i = e % d;
        float x = normed(e);
        if (v_from_k && head >= nq && vrow)     // the value is the key as projected, before norm and rotation
            vrow[(size_t)(head - nq) * page_size * dv + i] = qi::from_f32<T>(qi::to_f32<T>(row[e]) + (bias ? bias[e] : 0.f));
        if (i < rot) {
            int pair, other;
            bool first;
            if (interleaved) { pair = i >> 1; first = !(i & 1); other = first ? e + 1 : e - 1; }
            else { first = i < half; pair = first ? i : i - half; other = first ? e + half : e - half; }
            const float o = normed(other);
            float sn, cs;
            sincosf((float)pos * inv_freq[pair], &sn, &cs);
            x = first ? x * cs - o * sn : x * cs + o * sn;
        }
        if (head < nq) q_out[(size_t)t * nq * d + e] = qi::from_f32<T>(x * q_factor);
        else if (krow) krow[(size_t)(head - nq) * page_size * d + i] = qi::from_f32<T>(x);
    }
}

// The form for rows without biases and values from keys, in 16-byte pieces: LANES lanes a head (eight coordinates each, d <=
// 8 LANES), every operand read once. A warp takes 32 / LANES heads of q, k and v in turn. Norms of every head by itself, a
// rotation in neighbouring pairs (a lane holds whole pairs) and values mixed with another layer's are each optional.
template <typename T, int LANES>
__global__ void __launch_bounds__(256)
head_rope_kv_kernel(const T* __restrict__ proj, long long ld, T* __restrict__ q_out, const int* __restrict__ positions,
                    const int* __restrict__ token_req, const int* __restrict__ block_table, int max_blocks, int page_size,
                    int num_pages, T* __restrict__ k_pages, T* __restrict__ v_pages, int nq, int nkv, int d, int dv,
                    const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps, float temp_coef, int temp_every,
                    const float* __restrict__ inv_freq, int rot, const T* __restrict__ v_first, long long ldv, float v_share,
                    int n_tokens, int* __restrict__ status) {
    qi::pdl_wait();
    const int heads = nq + 2 * nkv, per_block = 256 / LANES;
    const int sub = threadIdx.x % LANES, i = sub * 8;
    const long long total = (long long)n_tokens * heads;
    for (long long it = (long long)blockIdx.x * per_block + threadIdx.x / LANES; it < (total + per_block - 1) / per_block * per_block;
         it += (long long)gridDim.x * per_block) {
        const bool in = it < total;           // whole warps stay together for the sums below
        const int t = in ? (int)(it / heads) : 0, hd = in ? (int)(it % heads) : 0;
        const bool is_v = hd >= nq + nkv;
        const int width = is_v ? dv : d;
        const T* src = proj + (size_t)t * ld + (is_v ? (size_t)(nq + nkv) * d + (size_t)(hd - nq - nkv) * dv : (size_t)hd * d);
        float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (in && i < width) qi::Vec8<T>::load(src + i, x);
        float sq = 0.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) sq = fmaf(x[j], x[j], sq);
#pragma unroll
        for (int o = LANES / 2; o > 0; o >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, o);
        if (!in || i >= width) continue;      // nothing below is collective
        const int pos = positions[t];
        if (pos < 0) {
            if (sub == 0 && status) atomicOr(status, qi::kStatusBadRange);
            continue;
        }
        T* dst;
        if (hd < nq) {
            dst = q_out + ((size_t)t * nq + hd) * d;
        } else {
            if (!k_pages) continue;
            const int page = block_table[(size_t)token_req[t] * max_blocks + pos / page_size];
            if (page < 0 || page >= num_pages) {
                if (sub == 0 && status) atomicOr(status, qi::kStatusBadPage);
                continue;
            }
            const int g = is_v ? hd - nq - nkv : hd - nq;
            dst = (is_v ? v_pages : k_pages) + (((size_t)page * nkv + g) * page_size + pos % page_size) * (size_t)width;
        }
        if (!is_v) {
            const float factor = hd < nq ? query_factor(pos, temp_coef, temp_every) : 1.f;
            if (q_gain) {
                float g[8];
                qi::Vec8<float>::load((hd < nq ? q_gain : k_gain) + i, g);
                const float inv = 1.0f / sqrtf(sq / (float)d + eps);
#pragma unroll
                for (int j = 0; j < 8; ++j) x[j] = x[j] * inv * g[j];
            }
#pragma unroll
            for (int j = 0; j < 8; j += 2) {
                if (i + j < rot) {
                    float sn, cs;
                    sincosf((float)pos * inv_freq[(i + j) >> 1], &sn, &cs);
                    const float u = x[j], v = x[j + 1];
                    x[j] = u * cs - v * sn;
                    x[j + 1] = v * cs + u * sn;
                }
            }
            if (temp_every > 0) {
#pragma unroll
                for (int j = 0; j < 8; ++j) x[j] *= factor;
            }
        } else if (v_first) {
            float f[8];
            qi::Vec8<T>::load(v_first + (size_t)t * ldv + (size_t)(hd - nq - nkv) * dv + i, f);
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] = (1.f - v_share) * x[j] + v_share * f[j];
        }
        qi::Vec8<T>::store(dst + i, x);
    }
}

}  // namespace

// q_gain, k_gain (both or neither; float32 [nq d], [nkv d]): q as a whole and k as a whole each pass an RMS norm with that
// gain and `eps` before the rotation; with head_norm every head by itself does, with a gain of d numbers that the heads
// share. temp_every > 0: q is multiplied by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1). v_first (or null; rows `ldv`
// elements apart, in `dtype`): a value v becomes (1 - v_share) v + v_share v_first before it is cached. v_from_k: the rows hold no v; a position's value is its key as projected (dv = d).
extern "C" int qi_norm_rope_kv_ex(const void* proj, long long ld, const float* bias, void* q_out, int dtype,
                               const float* inv_freq, int rot, int interleaved, const int* positions,
                               const int* token_req, const int* block_table, int max_blocks, int page_size,
                               int num_pages, void* k_pages, void* v_pages, int n_tokens, int nq, int nkv, int d,
                               int dv, const float* q_gain, const float* k_gain, float eps, int head_norm, int v_from_k, float temp_coef,
                               int temp_every, const void* v_first, long long ldv, float v_share, int* status, cudaStream_t stream) {
    QI_REQUIRE(!v_first || (!v_from_k && ldv >= (long long)nkv * dv), "bias_rope_kv: values to mix in need rows of values");
    QI_REQUIRE(n_tokens >= 0 && nq > 0 && nkv > 0 && d > 0 && dv > 0, "bias_rope_kv: bad sizes");
    QI_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= d, "bias_rope_kv: %d rotated coordinates do not fit a head of %d", rot, d);
    QI_REQUIRE(rot == 0 || inv_freq, "bias_rope_kv: a rotation needs its inverse frequencies");
    QI_REQUIRE((q_gain == nullptr) == (k_gain == nullptr) && (!q_gain || eps > 0.f), "bias_rope_kv: the norms of q and k come together, with a positive eps");
    QI_REQUIRE(!v_from_k || dv == d, "bias_rope_kv: values that are the keys have the keys' size");
    QI_REQUIRE(ld >= (long long)(nq + nkv) * d + (v_from_k ? 0 : (long long)nkv * dv), "bias_rope_kv: the rows are too short");
    QI_REQUIRE((k_pages == nullptr) == (v_pages == nullptr), "bias_rope_kv: key and value pages come together");
    QI_REQUIRE(!k_pages || (block_table && max_blocks > 0 && page_size > 0 && num_pages > 0), "bias_rope_kv: bad page geometry");
    QI_REQUIRE(nq + nkv <= 8192, "bias_rope_kv: too many heads");
    if (n_tokens == 0) return 0;
    if ((!q_gain || head_norm) && !bias && (!rot || interleaved) && !v_from_k && d % 8 == 0 && dv % 8 == 0 && d <= 256 && dv <= 256 && ld % 8 == 0 && ldv % 8 == 0 &&
        (((uintptr_t)proj | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)q_gain | (uintptr_t)k_gain | (uintptr_t)v_first) & 15) == 0) {
        const int wide = d > dv ? d : dv;
        const int lanes = wide <= 32 ? 4 : wide <= 64 ? 8 : wide <= 128 ? 16 : 32, per_block = 256 / lanes;
        long long blocks = ((long long)n_tokens * (nq + 2 * nkv) + per_block - 1) / per_block;
        if (blocks > 148 * 64) blocks = 148 * 64;
#define QI_HN(L)                                                                                                                     \
    qi::launch(head_rope_kv_kernel<T, L>, dim3((unsigned)blocks), dim3(256), 0, stream, (const T*)proj, ld, (T*)q_out, positions, token_req, \
               block_table, max_blocks, page_size, num_pages, (T*)k_pages, (T*)v_pages, nq, nkv, d, dv, q_gain, k_gain, eps, temp_coef, \
               temp_every, inv_freq, rot, (const T*)v_first, ldv, v_share, n_tokens, status)
        QI_DISPATCH_DTYPE(dtype, T, {
            if (lanes == 4) QI_HN(4);
            else if (lanes == 8) QI_HN(8);
            else if (lanes == 16) QI_HN(16);
            else QI_HN(32);
        });
#undef QI_HN
        return qi::check_launch("head_rope_kv");
    }
    QI_DISPATCH_DTYPE(dtype, T, {
        qi::launch(bias_rope_kv_kernel<T>, dim3(n_tokens), dim3(256), head_norm ? sizeof(float) * (nq + nkv) : 0, stream, (const T*)proj, ld, bias, (T*)q_out, inv_freq, rot,
                   interleaved, positions, token_req, block_table, max_blocks, page_size, num_pages, (T*)k_pages, (T*)v_pages,
                   nq, nkv, d, dv, q_gain, k_gain, eps, head_norm, v_from_k, temp_coef, temp_every,
                   (const T*)v_first, ldv, v_share, status);
    });
    return qi::check_launch("bias_rope_kv");
}

extern "C" int qi_bias_rope_kv(const void* proj, long long ld, const float* bias, void* q_out, int dtype,
                               const float* inv_freq, int rot, int interleaved, const int* positions,
                               const int* token_req, const int* block_table, int max_blocks, int page_size,
                               int num_pages, void* k_pages, void* v_pages, int n_tokens, int nq, int nkv, int d,
                               int dv, int* status, cudaStream_t stream) {
    return qi_norm_rope_kv_ex(proj, ld, bias, q_out, dtype, inv_freq, rot, interleaved, positions, token_req, block_table, max_blocks,
                           page_size, num_pages, k_pages, v_pages, n_tokens, nq, nkv, d, dv, nullptr, nullptr, 0.f, 0, 0, 0.f, 0, nullptr, 0, 0.f, status, stream);
}

// Causal grouped-query attention over the paged cache, for any span length,
// any head size up to 256 and any page size: the kernel of the true 32-bit
// path and the one that takes whatever the tensor-core kernels refuse.
//
// For the query of token t (request r, absolute position p) and query head h
// (kv head h / (nq / nkv): consecutive query heads share a kv head):
//     score_j = (sum_i q_i k_{j,i}) * scale          for lo <= j <= p
//     out     = sum_j softmax(score)_j * v_j
// with lo = 0, or p - window + 1 for a windowed layer, or the start of p's chunk
// (floor(p / chunk) * chunk, chunks counted from the sequence's first position)
// for a chunked layer; both bounds may hold at once, and the sequence's first `keep_first` keys may stay visible
// whatever those bounds say. A soft cap c replaces each
// score by c tanh(score / c) before the softmax; a distance bias then adds a number per
// head that depends on p - j alone. Values may have another
// size `dv` than queries and keys, and the result may be multiplied, element by
// element, by the sigmoid of a gate row (an output gate computed from the
// mixer's input). Scores, the maximum,
// the exponentials and the weighted sum are 32-bit. This is the reference's
// loop (crates/quantinfer-runtime/src/attention.rs:105-135; group :83,
// scale :84, causal bound :106,111) with the softmax evaluated online, one
// chunk of 32 keys at a time, so that no score row is stored.
//
// One block per (token, head); its four warps take chunks of keys in turn and
// their partial results are combined in warp order.
#include "common.cuh"

#include <math.h>

namespace {

constexpr int kWarps = 4;
constexpr int kMaxD = 256;
constexpr int kAccPerLane = kMaxD / 32;

template <typename T>
__global__ void __launch_bounds__(kWarps * 32)
attention_generic_kernel(const T* __restrict__ q, T* __restrict__ out, const T* __restrict__ k_pages,
                         const T* __restrict__ v_pages, const int* __restrict__ block_table,
                         int max_blocks, int page_size, int num_pages,
                         const int* __restrict__ positions, const int* __restrict__ token_req,
                         int nq, int nkv, int d, int dv, float scale, float softcap, float out_scale, int window, int chunk,
                         const T* __restrict__ gate, long long ldg, const float* __restrict__ sink, const float* __restrict__ bias, int bias_len,
                         long long ldo, int keep_first, int* __restrict__ status) {
    extern __shared__ float smem[];
    float* q_s = smem;                          // [d]
    float* part_acc = smem + d;                 // [kWarps][dv]
    float* part_m = part_acc + kWarps * dv;     // [kWarps]
    float* part_l = part_m + kWarps;            // [kWarps]

    qi::pdl_enter();
    const int t = blockIdx.y, h = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int hk = h / (nq / nkv);
    const int pos = positions[t];
    const int r = token_req[t];
    const int* table = block_table + (size_t)r * max_blocks;
    int lo = (window > 0 && pos - window + 1 > 0) ? pos - window + 1 : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    // the keys in one row of numbers: the kept first ones that lie before `lo`, then lo .. pos
    const int head = min(keep_first, lo), last = head + pos - lo;

    const T* qrow = q + ((size_t)t * nq + h) * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) q_s[i] = qi::to_f32<T>(qrow[i]);
    __syncthreads();

    float m = -INFINITY, l = 0.f;
    float acc[kAccPerLane];
#pragma unroll
    for (int i = 0; i < kAccPerLane; ++i) acc[i] = 0.f;

    bool bad_page = false;
    for (int base = warp * 32; base <= last; base += kWarps * 32) {
        const int at = base + lane, j = at < head ? at : lo + at - head;
        const bool valid = at <= last;
        float s = -INFINITY;
        if (valid) {
            const int page = table[j / page_size];
            if (page < 0 || page >= num_pages) {
                bad_page = true;
            } else {
                const T* krow = k_pages + (((size_t)page * nkv + hk) * page_size + (j % page_size)) * (size_t)d;
                float dot = 0.f;
                for (int i = 0; i < d; ++i) dot = fmaf(q_s[i], qi::to_f32<T>(krow[i]), dot);
                s = dot * scale;
                if (softcap > 0.f) s = softcap * tanhf(s / softcap);
                if (bias) s += bias[(size_t)h * bias_len + min(pos - j, bias_len - 1)];
            }
        }
        const float cm = qi::warp_max(s);
        if (cm == -INFINITY) continue;  // only after a bad page
        const float m_new = fmaxf(m, cm);
        const float corr = expf(m - m_new);  // m = -inf on the first chunk gives 0
        const float p = (s == -INFINITY) ? 0.f : expf(s - m_new);
        l = l * corr + qi::warp_sum(p);
#pragma unroll
        for (int i = 0; i < kAccPerLane; ++i) acc[i] *= corr;
        const int count = min(32, last - base + 1);
        for (int jj = 0; jj < count; ++jj) {
            const float pj = __shfl_sync(0xffffffffu, p, jj);
            const int key = base + jj < head ? base + jj : lo + base + jj - head;
            const int page = table[key / page_size];
            if (page < 0 || page >= num_pages) continue;
            const T* vrow = v_pages + (((size_t)page * nkv + hk) * page_size + (key % page_size)) * (size_t)dv;
#pragma unroll
            for (int i = 0; i < kAccPerLane; ++i) {
                const int idx = lane + 32 * i;
                if (idx < dv) acc[i] = fmaf(pj, qi::to_f32<T>(vrow[idx]), acc[i]);
            }
        }
        m = m_new;
    }
    if (bad_page && status) atomicOr(status, qi::kStatusBadPage);

    if (lane == 0) {
        part_m[warp] = m;
        part_l[warp] = l;
    }
#pragma unroll
    for (int i = 0; i < kAccPerLane; ++i) {
        const int idx = lane + 32 * i;
        if (idx < dv) part_acc[warp * dv + idx] = acc[i];
    }
    __syncthreads();

    float gm = sink ? sink[h] : -INFINITY;      // the sink: one more term in the denominator, with no key and no value
    for (int w = 0; w < kWarps; ++w) gm = fmaxf(gm, part_m[w]);
    float gl = 0.f;
    float wscale[kWarps];
    for (int w = 0; w < kWarps; ++w) {
        wscale[w] = (part_m[w] == -INFINITY) ? 0.f : expf(part_m[w] - gm);
        gl += part_l[w] * wscale[w];
    }
    if (sink) gl += expf(sink[h] - gm);
    T* orow = out + (size_t)t * ldo + (size_t)h * dv;
    const T* grow = gate ? gate + (size_t)t * ldg + (size_t)h * dv : nullptr;
    for (int i = threadIdx.x; i < dv; i += blockDim.x) {
        float o = 0.f;
        for (int w = 0; w < kWarps; ++w) o += part_acc[w * dv + i] * wscale[w];
        o = gl > 0.f ? o / gl : 0.f;
        if (grow) o = o / (1.0f + expf(-qi::to_f32<T>(grow[i])));
        o *= out_scale;
        orow[i] = qi::from_f32<T>(o);
    }
}

}  // namespace

// q [n, nq d]; out [n, nq dv]; k_pages [pages, nkv, page_size, d]; v_pages [pages, nkv, page_size, dv];
// window 0: no window; chunk 0: no chunks; gate (may be null): row t, head h, element i at gate[t * ldg + h * dv + i];
// softcap c > 0: a score s becomes c tanh(s / c) before the softmax (0: scores as they are); out_scale multiplies the result.
// sink (may be null): float32 [nq]; the softmax's denominator of head h holds exp(sink[h]) once more.
// bias (may be null): float32 [nq, bias_len]; a key n positions back adds bias[h, min(n, bias_len - 1)] to its score.
// ldo: elements from one row of out to the next. keep_first: keys 0 .. keep_first - 1 stay visible behind a window or chunk.
extern "C" int qi_attention_generic_bias(const void* q, void* out, int dtype, const void* k_pages,
                                       const void* v_pages, const int* block_table, int max_blocks,
                                       int page_size, int num_pages, const int* positions,
                                       const int* token_req, int n_tokens, int nq, int nkv, int d, int dv,
                                       float scale, float softcap, float out_scale, int window, int chunk, const void* gate,
                                       long long ldg, const float* sink, const float* bias, int bias_len, long long ldo,
                                       int keep_first, int* status, cudaStream_t stream) {
    QI_REQUIRE(keep_first >= 0, "attention: keep_first must be >= 0 (0 = none)");
    QI_REQUIRE(ldo >= (long long)nq * dv, "attention: the output's rows are too short");
    QI_REQUIRE(!bias || bias_len > 0, "attention: an empty distance bias");
    QI_REQUIRE(n_tokens >= 0 && nq > 0 && nkv > 0 && d > 0 && dv > 0, "attention: bad sizes");
    QI_REQUIRE(nq % nkv == 0, "attention: %d query heads are not a multiple of %d kv heads", nq, nkv);
    QI_REQUIRE(d <= kMaxD && dv <= kMaxD, "attention: head sizes %d / %d are above the limit %d of this kernel", d, dv, kMaxD);
    QI_REQUIRE(page_size > 0 && max_blocks > 0 && num_pages > 0, "attention: bad page geometry");
    QI_REQUIRE(window >= 0 && chunk >= 0, "attention: window and chunk must be >= 0 (0 = none)");
    QI_REQUIRE(softcap >= 0.f, "attention: the soft cap must be >= 0 (0 = none)");
    QI_REQUIRE(!gate || ldg >= (long long)nq * dv, "attention: the gate's rows are too short");
    QI_REQUIRE(n_tokens <= 65535 * 32768 && nq <= 65535, "attention: grid too large");
    if (n_tokens == 0) return 0;
    const size_t smem = sizeof(float) * ((size_t)d + kWarps * dv + 2 * kWarps);
    // grid.y is limited to 65535: launch in slabs of tokens.
    for (int t0 = 0; t0 < n_tokens; t0 += 65535) {
        const int nt = n_tokens - t0 < 65535 ? n_tokens - t0 : 65535;
        dim3 grid(nq, nt);
        QI_DISPATCH_DTYPE(dtype, T, {
            qi::launch(attention_generic_kernel<T>, grid, dim3(kWarps * 32), smem, stream,
                (const T*)q + (size_t)t0 * nq * d, (T*)out + (size_t)t0 * ldo, (const T*)k_pages,
                (const T*)v_pages, block_table, max_blocks, page_size, num_pages, positions + t0,
                token_req + t0, nq, nkv, d, dv, scale, softcap, out_scale, window, chunk,
                gate ? (const T*)gate + (size_t)t0 * ldg : (const T*)nullptr, ldg, sink, bias, bias_len, ldo, keep_first, status);
        });
    }
    return qi::check_launch("attention_generic");
}

extern "C" int qi_attention_generic_sink(const void* q, void* out, int dtype, const void* k_pages,
                                       const void* v_pages, const int* block_table, int max_blocks,
                                       int page_size, int num_pages, const int* positions,
                                       const int* token_req, int n_tokens, int nq, int nkv, int d, int dv,
                                       float scale, float softcap, float out_scale, int window, int chunk, const void* gate,
                                       long long ldg, const float* sink, int* status, cudaStream_t stream) {
    return qi_attention_generic_bias(q, out, dtype, k_pages, v_pages, block_table, max_blocks, page_size, num_pages, positions,
                                     token_req, n_tokens, nq, nkv, d, dv, scale, softcap, out_scale, window, chunk, gate, ldg,
                                     sink, nullptr, 0, (long long)nq * dv, 0, status, stream);
}

extern "C" int qi_attention_generic_cap(const void* q, void* out, int dtype, const void* k_pages,
                                       const void* v_pages, const int* block_table, int max_blocks,
                                       int page_size, int num_pages, const int* positions,
                                       const int* token_req, int n_tokens, int nq, int nkv, int d, int dv,
                                       float scale, float softcap, float out_scale, int window, int chunk, const void* gate,
                                       long long ldg, int* status, cudaStream_t stream) {
    return qi_attention_generic_sink(q, out, dtype, k_pages, v_pages, block_table, max_blocks, page_size, num_pages, positions,
                                     token_req, n_tokens, nq, nkv, d, dv, scale, softcap, out_scale, window, chunk, gate, ldg,
                                     nullptr, status, stream);
}

extern "C" int qi_attention_generic_ex(const void* q, void* out, int dtype, const void* k_pages,
                                       const void* v_pages, const int* block_table, int max_blocks,
                                       int page_size, int num_pages, const int* positions,
                                       const int* token_req, int n_tokens, int nq, int nkv, int d, int dv,
                                       float scale, int window, int chunk, const void* gate, long long ldg,
                                       int* status, cudaStream_t stream) {
    return qi_attention_generic_cap(q, out, dtype, k_pages, v_pages, block_table, max_blocks, page_size, num_pages, positions,
                                    token_req, n_tokens, nq, nkv, d, dv, scale, 0.f, 1.f, window, chunk, gate, ldg, status, stream);
}

extern "C" int qi_attention_generic(const void* q, void* out, int dtype, const void* k_pages,
                                    const void* v_pages, const int* block_table, int max_blocks,
                                    int page_size, int num_pages, const int* positions,
                                    const int* token_req, int n_tokens, int nq, int nkv, int d,
                                    float scale, int window, int* status, cudaStream_t stream) {
    return qi_attention_generic_ex(q, out, dtype, k_pages, v_pages, block_table, max_blocks, page_size, num_pages, positions,
                                   token_req, n_tokens, nq, nkv, d, d, scale, window, 0, nullptr, 0, status, stream);
}

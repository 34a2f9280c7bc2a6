// Residual streams that are mixed at every sublayer (hyper-connections). A token has S streams x_0 .. x_(S-1) of `width`
// 32-bit numbers, side by side in one row. One kernel does what lies between two sublayers:
//
//     x_t <- sum_s mix[s, t] x_s + share[t] y            all streams at once, y the result of the sublayer before
//     u   =  sum_t in[t] x_t                             what the next sublayer reads (in null: the plain sum)
//     out =  norm(u)                                     layer norm or RMS norm with gain (and bias), in the activation type
//
// y comes whole or as the partial sums of a product whose contraction was split (added in order); without y the streams
// stay as they are; without `out` only the streams move on. With `rows` the source rows are gathered and nothing is
// written back. All arithmetic is 32-bit; mix, share and in are read from device memory.
#include "common.cuh"
#include "vec8.cuh"

namespace {

using qi::Vec8;
constexpr int kMaxStreams = 16;

// A row in registers: eight neighbouring coordinates of every stream a thread, every operand read once. A CTA takes rows
// blockIdx.x, blockIdx.x + gridDim.x, ...
template <typename TD, typename TO, int S>
__global__ void __launch_bounds__(512, S <= 2 ? 2 : 1)
hyper_norm_vec_kernel(float* __restrict__ streams, const TD* __restrict__ y, int y_splits, size_t y_split_stride,
                      const float* __restrict__ mix, const float* __restrict__ share, const float* __restrict__ in,
                      const float* __restrict__ gain, const float* __restrict__ bias, float eps, int center, TO* __restrict__ out,
                      const int* __restrict__ rows, int width, int write_back, int n_rows) {
    __shared__ float scratch[32];
    qi::pdl_wait();
    const int i = threadIdx.x * 8;
    const bool active = i < width;
    float m[S][S], w_out[S], w_in[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
#pragma unroll
        for (int t = 0; t < S; ++t) m[s][t] = y ? mix[s * S + t] : 0.f;
        w_out[s] = y ? share[s] : 0.f;
        w_in[s] = in ? in[s] : 1.f;
    }
    for (int r = blockIdx.x; r < n_rows; r += gridDim.x) {
        const int src = rows ? rows[r] : r;
        float* row = streams + (size_t)src * S * width;
        float u[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, g[8], b[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (active) {
            float x[S][8];
#pragma unroll
            for (int s = 0; s < S; ++s) Vec8<float>::load(row + (size_t)s * width + i, x[s]);
            if (out) {
                Vec8<float>::load(gain + i, g);
                if (bias) Vec8<float>::load(bias + i, b);
            }
            if (y) {
                float acc[8], d[8];
                const TD* yr = y + (size_t)src * width + i;
                Vec8<TD>::load(yr, acc);
#pragma unroll 4
                for (int k = 1; k < y_splits; ++k) {
                    Vec8<TD>::load(yr + k * y_split_stride, d);
#pragma unroll
                    for (int j = 0; j < 8; ++j) acc[j] += d[j];
                }
#pragma unroll
                for (int j = 0; j < 8; ++j) {
                    float next[S];
#pragma unroll
                    for (int t = 0; t < S; ++t) {
                        float v = w_out[t] * acc[j];
#pragma unroll
                        for (int s = 0; s < S; ++s) v = fmaf(m[s][t], x[s][j], v);
                        next[t] = v;
                    }
#pragma unroll
                    for (int t = 0; t < S; ++t) x[t][j] = next[t];
                }
                if (write_back) {
#pragma unroll
                    for (int s = 0; s < S; ++s) Vec8<float>::store(row + (size_t)s * width + i, x[s]);
                }
            }
#pragma unroll
            for (int j = 0; j < 8; ++j) {
#pragma unroll
                for (int s = 0; s < S; ++s) u[j] = fmaf(w_in[s], x[s][j], u[j]);
            }
        }
        if (!out) continue;
        float mean = 0.f;
        if (center) {
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < 8; ++j) sum += u[j];
            mean = qi::block_sum(sum, scratch) / (float)width;
        }
        float sq = 0.f;
        if (active) {
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                u[j] -= mean;
                sq = fmaf(u[j], u[j], sq);
            }
        }
        const float inv = 1.0f / sqrtf(qi::block_sum(sq, scratch) / (float)width + eps);
        if (active) {
#pragma unroll
            for (int j = 0; j < 8; ++j) u[j] = fmaf(u[j] * inv, g[j], b[j]);
            Vec8<TO>::store(out + (size_t)r * width + i, u);
        }
    }
}

// Any width and up to kMaxStreams streams: a coordinate at a time, u in shared memory between the passes.
template <typename TD, typename TO>
__global__ void hyper_norm_kernel(float* __restrict__ streams, const TD* __restrict__ y, int y_splits, size_t y_split_stride,
                                  const float* __restrict__ mix, const float* __restrict__ share, const float* __restrict__ in,
                                  const float* __restrict__ gain, const float* __restrict__ bias, float eps, int center,
                                  TO* __restrict__ out, const int* __restrict__ rows, int n_streams, int width, int write_back) {
    extern __shared__ float u_row[];         // [width]
    __shared__ float scratch[32];
    qi::pdl_wait();
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    float* row = streams + (size_t)src * n_streams * width;
    float sum = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        float x[kMaxStreams], u = 0.f, acc = 0.f;
        for (int s = 0; s < n_streams; ++s) x[s] = row[(size_t)s * width + i];
        if (y) {
            for (int k = 0; k < y_splits; ++k) acc += qi::to_f32<TD>(y[k * y_split_stride + (size_t)src * width + i]);
        }
        for (int t = 0; t < n_streams; ++t) {
            float v = x[t];
            if (y) {
                v = share[t] * acc;
                for (int s = 0; s < n_streams; ++s) v = fmaf(mix[s * n_streams + t], x[s], v);
                if (write_back) row[(size_t)t * width + i] = v;     // this thread holds every old number of this coordinate
            }
            u = fmaf(in ? in[t] : 1.f, v, u);
        }
        if (out) u_row[i] = u;
        sum += u;
    }
    if (!out) return;
    const float mean = center ? qi::block_sum(sum, scratch) / (float)width : 0.f;
    float sq = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float d = u_row[i] - mean;
        sq = fmaf(d, d, sq);
    }
    const float inv = 1.0f / sqrtf(qi::block_sum(sq, scratch) / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x)
        out[(size_t)r * width + i] = qi::from_f32<TO>(fmaf((u_row[i] - mean) * inv, gain[i], bias ? bias[i] : 0.f));
}

}  // namespace

extern "C" int qi_hyper_max_streams() { return kMaxStreams; }

// streams float32 [*, n_streams, width]; y (or null) [y_splits, rows of streams, width] in `y_dtype`; mix float32
// [n_streams, n_streams] ([from, to]) and share float32 [n_streams], needed with y; in float32 [n_streams] or null (ones);
// out [n_rows, width] in `out_dtype` or null; gain float32 [width] (needed with out), bias float32 [width] or null; center 1:
// layer norm, 0: RMS norm. rows (or null): the source row of every output row; write_back must be 0 then.
extern "C" int qi_hyper_norm(float* streams, const void* y, int y_dtype, int y_splits, long long y_split_stride, const float* mix,
                             const float* share, const float* in, const float* gain, const float* bias, float eps, int center,
                             void* out, int out_dtype, const int* rows, int n_rows, int n_streams, int width, int write_back,
                             cudaStream_t stream) {
    QI_REQUIRE(n_rows >= 0 && width > 0 && n_streams >= 1 && n_streams <= kMaxStreams, "hyper_norm: bad sizes rows=%d width=%d streams=%d (1..%d)",
               n_rows, width, n_streams, kMaxStreams);
    QI_REQUIRE(!y || (mix && share && y_splits >= 1), "hyper_norm: a sublayer's result needs its mix and its shares");
    QI_REQUIRE(!out || (gain && eps > 0.f), "hyper_norm: the norm's gain is missing or eps is not positive");
    QI_REQUIRE(!(rows && write_back), "hyper_norm: the row-gather form does not write the streams");
    if (n_rows == 0 || (!out && !(y && write_back))) return 0;
    const int dd = y ? y_dtype : qi::kF32, od = out ? out_dtype : qi::kF32;
    const bool vec = n_streams <= 4 && width % 8 == 0 && width <= 4096 && ((uintptr_t)streams & 31) == 0 &&
                     (((uintptr_t)y | (uintptr_t)out | (uintptr_t)gain | (uintptr_t)bias) & 15) == 0 && y_split_stride % 8 == 0;
    if (vec) {
        const int threads = (width / 8 + 31) / 32 * 32;
        const int resident = 148 * (1024 / threads < 16 ? 1024 / threads : 16);
        const int grid = n_rows < resident ? n_rows : resident;
#define QI_HY(S)                                                                                                                   \
    qi::launch(hyper_norm_vec_kernel<TD, TO, S>, dim3(grid), dim3(threads), 0, stream, streams, (const TD*)y, y_splits,             \
               (size_t)y_split_stride, mix, share, in, gain, bias, eps, center, (TO*)out, rows, width, write_back, n_rows)
        QI_DISPATCH_DTYPE(dd, TD, {
            QI_DISPATCH_DTYPE(od, TO, {
                if (n_streams == 1) QI_HY(1);
                else if (n_streams == 2) QI_HY(2);
                else if (n_streams == 3) QI_HY(3);
                else QI_HY(4);
            });
        });
#undef QI_HY
        return qi::check_launch("hyper_norm");
    }
    const size_t smem = out ? sizeof(float) * (size_t)width : 0;
    QI_REQUIRE(smem <= 200 * 1024, "hyper_norm: rows of %d numbers do not fit this kernel (51200)", width);
    const int threads = width >= 2048 ? 512 : (width >= 512 ? 256 : (width >= 128 ? 128 : 32));
    QI_DISPATCH_DTYPE(dd, TD, {
        QI_DISPATCH_DTYPE(od, TO, {
            if (smem > 48 * 1024) {
                const cudaError_t e = cudaFuncSetAttribute(hyper_norm_kernel<TD, TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
                QI_REQUIRE(e == cudaSuccess, "hyper_norm: cannot reserve %d bytes of shared memory: %s", (int)smem, cudaGetErrorString(e));
            }
            qi::launch(hyper_norm_kernel<TD, TO>, dim3(n_rows), dim3(threads), smem, stream, streams, (const TD*)y, y_splits,
                       (size_t)y_split_stride, mix, share, in, gain, bias, eps, center, (TO*)out, rows, n_streams, width, write_back);
        });
    });
    return qi::check_launch("hyper_norm");
}

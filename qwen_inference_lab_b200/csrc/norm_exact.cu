// Root-mean-square norm whose arithmetic is float32 from end to end, for residual streams that are
// kept in float32 whatever the activation dtype is.
//
//   y = x / sqrt(mean(x^2) + eps) * (offset + w)
//
// Input and output types are independent (a float32 stream normed into bfloat16 rows for the
// products that follow); the statistics, the scaling and the weight multiply are float32 and the
// result is rounded once.  `offset` 1 serves weights that are stored around zero, 0 plain ones.
// With `rows` only those rows are normed, in that order.  The sum of squares is taken by a fixed
// tree over a fixed block size, so a row's result does not depend on the rest of the batch.
#include "common.cuh"

template <typename TI, typename TO, typename W>
__global__ void __launch_bounds__(256)
rmsnorm_exact_kernel(const TI* __restrict__ x, const W* __restrict__ weight, const int* __restrict__ rows,
                     TO* __restrict__ out, int width, float eps, float offset, long long ld) {
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const int r = blockIdx.x;
    const TI* src = x + (size_t)(rows ? rows[r] : r) * (size_t)ld;      // ld: the input's row stride (a column range of a wider buffer)
    TO* dst = out + (size_t)r * width;
    float sq = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        const float v = to_f32<TI>(src[i]);
        sq = fmaf(v, v, sq);
    }
    sq = block_sum(sq, scratch);
    const float scale = 1.0f / sqrtf(sq / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += 256)
        dst[i] = from_f32<TO>(to_f32<TI>(src[i]) * scale * (offset + to_f32<W>(weight[i])));
}

extern "C" int qil_rmsnorm_exact(const void* x, int x_dtype, const void* weight, int weight_dtype, const int* rows,
                                 void* out, int out_dtype, int n_rows, int width, float eps, float offset,
                                 long long ld, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0 || ld < width) QIL_REFUSE("rmsnorm_exact: width %d, row stride %lld", width, ld);
#define QIL_NORM_GO(TI, TO)                                                                                  \
    do {                                                                                                     \
        if (weight_dtype == QIL_F32)                                                                         \
            qil_launch_chained(rmsnorm_exact_kernel<TI, TO, float>, dim3(n_rows), dim3(256), 0, stream,      \
                               (const TI*)x, (const float*)weight, rows, (TO*)out, width, eps, offset, ld);  \
        else                                                                                                 \
            qil_launch_chained(rmsnorm_exact_kernel<TI, TO, bf16>, dim3(n_rows), dim3(256), 0, stream,       \
                               (const TI*)x, (const bf16*)weight, rows, (TO*)out, width, eps, offset, ld);   \
    } while (0)
    if (weight_dtype != QIL_F32 && weight_dtype != QIL_BF16) QIL_REFUSE("rmsnorm_exact: weight dtype %d", weight_dtype);
    if (x_dtype == QIL_F32 && out_dtype == QIL_F32) QIL_NORM_GO(float, float);
    else if (x_dtype == QIL_F32 && out_dtype == QIL_BF16) QIL_NORM_GO(float, bf16);
    else if (x_dtype == QIL_BF16 && out_dtype == QIL_BF16) QIL_NORM_GO(bf16, bf16);
    else if (x_dtype == QIL_BF16 && out_dtype == QIL_F32) QIL_NORM_GO(bf16, float);
    else QIL_REFUSE("rmsnorm_exact: dtypes %d -> %d", x_dtype, out_dtype);
#undef QIL_NORM_GO
    QIL_CHECK_LAUNCH();
}

// Layer norm with weight and bias (null: none), float32 from end to end like the norm above:
//
//   y = (x - mean) / sqrt(var + eps) * w + b,     var = mean((x - mean)^2)
//
// Two passes over the row (the mean, then the squared deviations from it), each a fixed tree.
template <typename TI, typename TO, typename W>
__global__ void __launch_bounds__(256)
layernorm_exact_kernel(const TI* __restrict__ x, const W* __restrict__ weight, const W* __restrict__ bias,
                       const int* __restrict__ rows, TO* __restrict__ out, int width, float eps) {
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const int r = blockIdx.x;
    const TI* src = x + (size_t)(rows ? rows[r] : r) * width;
    TO* dst = out + (size_t)r * width;
    float sum = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) sum += to_f32<TI>(src[i]);
    const float mean = block_sum(sum, scratch) / (float)width;
    float sq = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        const float v = to_f32<TI>(src[i]) - mean;
        sq = fmaf(v, v, sq);
    }
    sq = block_sum(sq, scratch);
    const float scale = 1.0f / sqrtf(sq / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += 256)
        dst[i] = from_f32<TO>((to_f32<TI>(src[i]) - mean) * scale * to_f32<W>(weight[i]) + (bias != nullptr ? to_f32<W>(bias[i]) : 0.f));
}

extern "C" int qil_layernorm_exact(const void* x, int x_dtype, const void* weight, const void* bias, int weight_dtype,
                                   const int* rows, void* out, int out_dtype, int n_rows, int width, float eps,
                                   cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0) QIL_REFUSE("layernorm_exact: width %d", width);
#define QIL_NORM_GO(TI, TO)                                                                                    \
    do {                                                                                                       \
        if (weight_dtype == QIL_F32)                                                                           \
            qil_launch_chained(layernorm_exact_kernel<TI, TO, float>, dim3(n_rows), dim3(256), 0, stream,      \
                               (const TI*)x, (const float*)weight, (const float*)bias, rows, (TO*)out, width, eps); \
        else                                                                                                   \
            qil_launch_chained(layernorm_exact_kernel<TI, TO, bf16>, dim3(n_rows), dim3(256), 0, stream,       \
                               (const TI*)x, (const bf16*)weight, (const bf16*)bias, rows, (TO*)out, width, eps); \
    } while (0)
    if (weight_dtype != QIL_F32 && weight_dtype != QIL_BF16) QIL_REFUSE("layernorm_exact: weight dtype %d", weight_dtype);
    if (x_dtype == QIL_F32 && out_dtype == QIL_F32) QIL_NORM_GO(float, float);
    else if (x_dtype == QIL_F32 && out_dtype == QIL_BF16) QIL_NORM_GO(float, bf16);
    else if (x_dtype == QIL_BF16 && out_dtype == QIL_BF16) QIL_NORM_GO(bf16, bf16);
    else if (x_dtype == QIL_BF16 && out_dtype == QIL_F32) QIL_NORM_GO(bf16, float);
    else QIL_REFUSE("layernorm_exact: dtypes %d -> %d", x_dtype, out_dtype);
#undef QIL_NORM_GO
    QIL_CHECK_LAUNCH();
}

// x += y / sqrt(mean(y^2) + eps) * w: a branch that is normed by its own root mean square before it joins the
// residual stream.  float32 arithmetic; x is the stream (float32 or bfloat16), y the branch.
template <typename TX, typename TY, typename W>
__global__ void __launch_bounds__(256)
rms_scale_add_kernel(TX* __restrict__ x, const TY* __restrict__ y, const W* __restrict__ weight, int width, float eps) {
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const TY* src = y + (size_t)blockIdx.x * width;
    TX* dst = x + (size_t)blockIdx.x * width;
    float sq = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        const float v = to_f32<TY>(src[i]);
        sq = fmaf(v, v, sq);
    }
    sq = block_sum(sq, scratch);
    const float scale = 1.0f / sqrtf(sq / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += 256)
        dst[i] = from_f32<TX>(to_f32<TX>(dst[i]) + to_f32<TY>(src[i]) * scale * to_f32<W>(weight[i]));
}

extern "C" int qil_rms_scale_add(void* x, int x_dtype, const void* y, int y_dtype, const void* weight, int weight_dtype,
                                 int n_rows, int width, float eps, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0) QIL_REFUSE("rms_scale_add: width %d", width);
#define QIL_NORM_GO(TX, TY)                                                                                   \
    do {                                                                                                      \
        if (weight_dtype == QIL_F32)                                                                          \
            qil_launch_chained(rms_scale_add_kernel<TX, TY, float>, dim3(n_rows), dim3(256), 0, stream,       \
                               (TX*)x, (const TY*)y, (const float*)weight, width, eps);                       \
        else                                                                                                  \
            qil_launch_chained(rms_scale_add_kernel<TX, TY, bf16>, dim3(n_rows), dim3(256), 0, stream,        \
                               (TX*)x, (const TY*)y, (const bf16*)weight, width, eps);                        \
    } while (0)
    if (weight_dtype != QIL_F32 && weight_dtype != QIL_BF16) QIL_REFUSE("rms_scale_add: weight dtype %d", weight_dtype);
    if (x_dtype == QIL_F32 && y_dtype == QIL_F32) QIL_NORM_GO(float, float);
    else if (x_dtype == QIL_F32 && y_dtype == QIL_BF16) QIL_NORM_GO(float, bf16);
    else if (x_dtype == QIL_BF16 && y_dtype == QIL_BF16) QIL_NORM_GO(bf16, bf16);
    else if (x_dtype == QIL_BF16 && y_dtype == QIL_F32) QIL_NORM_GO(bf16, float);
    else QIL_REFUSE("rms_scale_add: dtypes %d += %d", x_dtype, y_dtype);
#undef QIL_NORM_GO
    QIL_CHECK_LAUNCH();
}

// A branch joins the stream through a norm on the branch: x += mult * rms(a; w), rms(a; w) = a / sqrt(mean(a^2) + eps) * w.
// With a second branch b the two are first normed with weights of their own and averaged:
//   y = pre * (rms(a; wa) + rms(b; wb)),   x += mult * rms(y; w).
// float32 arithmetic throughout; x is the stream (float32 or bfloat16), a and b share a type.
template <typename TX, typename TA, typename W>
__global__ void __launch_bounds__(256)
rms_join_kernel(TX* __restrict__ x, const TA* __restrict__ a, const W* __restrict__ wa, const TA* __restrict__ b,
                const W* __restrict__ wb, const W* __restrict__ w, int width, float eps, float pre, float mult,
                bf16* __restrict__ rows) {
    // rows: null, or [N, width]: the stream's new values once more, rounded to bfloat16 (what the next product reads)
    extern __shared__ float y[];             // [width] when there are two branches
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const TA* ra = a + (size_t)blockIdx.x * width;
    TX* dst = x + (size_t)blockIdx.x * width;
    bf16* copy = rows != nullptr ? rows + (size_t)blockIdx.x * width : nullptr;
    float sa = 0.f, sb = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        const float v = to_f32<TA>(ra[i]);
        sa = fmaf(v, v, sa);
    }
    sa = block_sum(sa, scratch);
    const float scale_a = 1.0f / sqrtf(sa / (float)width + eps);
    if (b == nullptr) {
        for (int i = threadIdx.x; i < width; i += 256) {
            const TX next = from_f32<TX>(to_f32<TX>(dst[i]) + mult * (to_f32<TA>(ra[i]) * scale_a * to_f32<W>(w[i])));
            dst[i] = next;
            if (copy != nullptr) copy[i] = from_f32<bf16>(to_f32<TX>(next));
        }
        return;
    }
    const TA* rb = b + (size_t)blockIdx.x * width;
    for (int i = threadIdx.x; i < width; i += 256) {
        const float v = to_f32<TA>(rb[i]);
        sb = fmaf(v, v, sb);
    }
    sb = block_sum(sb, scratch);
    const float scale_b = 1.0f / sqrtf(sb / (float)width + eps);
    float sy = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        const float v = pre * (to_f32<TA>(ra[i]) * scale_a * to_f32<W>(wa[i]) + to_f32<TA>(rb[i]) * scale_b * to_f32<W>(wb[i]));
        y[i] = v;
        sy = fmaf(v, v, sy);
    }
    sy = block_sum(sy, scratch);
    const float scale_y = 1.0f / sqrtf(sy / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += 256) {       // a thread reads back what it wrote itself
        const TX next = from_f32<TX>(to_f32<TX>(dst[i]) + mult * (y[i] * scale_y * to_f32<W>(w[i])));
        dst[i] = next;
        if (copy != nullptr) copy[i] = from_f32<bf16>(to_f32<TX>(next));
    }
}

extern "C" int qil_rms_join(void* x, int x_dtype, const void* a, const void* wa, const void* b, const void* wb,
                            int branch_dtype, const void* w, int weight_dtype, int n_rows, int width, float eps,
                            float pre, float mult, void* rows, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0 || width > 40960) QIL_REFUSE("rms_join: width %d", width);
    if (b != nullptr && (wa == nullptr || wb == nullptr)) QIL_REFUSE("rms_join: two branches need a weight each");
    const size_t smem = b != nullptr ? (size_t)width * sizeof(float) : 0;
    cudaError_t err = cudaSuccess;
#define QIL_JOIN_GO(TX, TA, WT)                                                                                   \
    do {                                                                                                          \
        if (smem > 48 * 1024)                                                                                     \
            err = cudaFuncSetAttribute(rms_join_kernel<TX, TA, WT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (err == cudaSuccess)                                                                                   \
            qil_launch_chained(rms_join_kernel<TX, TA, WT>, dim3(n_rows), dim3(256), smem, stream, (TX*)x,        \
                               (const TA*)a, (const WT*)wa, (const TA*)b, (const WT*)wb, (const WT*)w, width, eps, \
                               pre, mult, (bf16*)rows);                                                           \
    } while (0)
#define QIL_JOIN_W(TX, TA)                                                                                        \
    do {                                                                                                          \
        if (weight_dtype == QIL_F32) QIL_JOIN_GO(TX, TA, float); else QIL_JOIN_GO(TX, TA, bf16);                  \
    } while (0)
    if (weight_dtype != QIL_F32 && weight_dtype != QIL_BF16) QIL_REFUSE("rms_join: weight dtype %d", weight_dtype);
    if (x_dtype == QIL_F32 && branch_dtype == QIL_F32) QIL_JOIN_W(float, float);
    else if (x_dtype == QIL_F32 && branch_dtype == QIL_BF16) QIL_JOIN_W(float, bf16);
    else if (x_dtype == QIL_BF16 && branch_dtype == QIL_BF16) QIL_JOIN_W(bf16, bf16);
    else if (x_dtype == QIL_BF16 && branch_dtype == QIL_F32) QIL_JOIN_W(bf16, float);
    else QIL_REFUSE("rms_join: dtypes %d += %d", x_dtype, branch_dtype);
#undef QIL_JOIN_W
#undef QIL_JOIN_GO
    if (err != cudaSuccess) { snprintf(qil_error_text, sizeof(qil_error_text), "%s", cudaGetErrorString(err)); return (int)err; }
    QIL_CHECK_LAUNCH();
}

// A branch joins the stream through a norm on the branch, and the next sublayer's norm of the new stream rides along:
//   x += norm(a; w),   rows = norm(x; next_w)          (rows and next_w are optional; rows without next_w: x rounded)
// where norm is the root-mean-square norm (center 0) or the layer norm without a bias (center 1: the mean is taken
// off first, the variance is the mean of the squared deviations).  float32 arithmetic, every reduction a fixed tree
// over one row; x is the stream (float32 or bfloat16), a the branch (float32), rows what the next product reads.
template <typename TX, typename W, typename TO>
__global__ void __launch_bounds__(256)
norm_join_kernel(TX* __restrict__ x, const float* __restrict__ a, const W* __restrict__ w, int width, float eps, int center,
                 const W* __restrict__ next_w, float next_eps, int next_center, TO* __restrict__ rows) {
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const float* ra = a + (size_t)blockIdx.x * width;
    TX* dst = x + (size_t)blockIdx.x * width;
    float mean = 0.f;
    if (center) {
        float sum = 0.f;
        for (int i = threadIdx.x; i < width; i += 256) sum += ra[i];
        mean = block_sum(sum, scratch) / (float)width;
    }
    float sq = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        const float v = ra[i] - mean;
        sq = fmaf(v, v, sq);
    }
    sq = block_sum(sq, scratch);
    const float scale = 1.0f / sqrtf(sq / (float)width + eps);
    float sum = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {       // a thread reads back below what it wrote itself
        const TX next = from_f32<TX>(to_f32<TX>(dst[i]) + (ra[i] - mean) * scale * to_f32<W>(w[i]));
        dst[i] = next;
        sum += to_f32<TX>(next);
    }
    if (rows == nullptr) return;
    TO* out = rows + (size_t)blockIdx.x * width;
    if (next_w == nullptr) {
        for (int i = threadIdx.x; i < width; i += 256) out[i] = from_f32<TO>(to_f32<TX>(dst[i]));
        return;
    }
    mean = 0.f;
    if (next_center) mean = block_sum(sum, scratch) / (float)width;
    sq = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        const float v = to_f32<TX>(dst[i]) - mean;
        sq = fmaf(v, v, sq);
    }
    sq = block_sum(sq, scratch);
    const float next_scale = 1.0f / sqrtf(sq / (float)width + next_eps);
    for (int i = threadIdx.x; i < width; i += 256)
        out[i] = from_f32<TO>((to_f32<TX>(dst[i]) - mean) * next_scale * to_f32<W>(next_w[i]));
}

// The same with the row held in registers (rows of up to 256 * VPT values): the branch and the stream are read once,
// every value is summed in the order the kernel above sums it, so both give the same bits.
template <typename TX, typename W, typename TO, int VPT>
__global__ void __launch_bounds__(256)
norm_join_regs_kernel(TX* __restrict__ x, const float* __restrict__ a, const W* __restrict__ w, int width, float eps, int center,
                      const W* __restrict__ next_w, float next_eps, int next_center, TO* __restrict__ rows) {
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const float* ra = a + (size_t)blockIdx.x * width;
    TX* dst = x + (size_t)blockIdx.x * width;
    float va[VPT], vx[VPT];
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int i = threadIdx.x + k * 256;
        va[k] = i < width ? ra[i] : 0.f;
        if (i < width) sum += va[k];
    }
    float mean = 0.f;
    if (center) mean = block_sum(sum, scratch) / (float)width;
    float sq = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k)
        if (threadIdx.x + k * 256 < width) { const float v = va[k] - mean; sq = fmaf(v, v, sq); }
    sq = block_sum(sq, scratch);
    const float scale = 1.0f / sqrtf(sq / (float)width + eps);
    sum = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int i = threadIdx.x + k * 256;
        vx[k] = 0.f;
        if (i < width) {
            const TX next = from_f32<TX>(to_f32<TX>(dst[i]) + (va[k] - mean) * scale * to_f32<W>(w[i]));
            dst[i] = next;
            vx[k] = to_f32<TX>(next);
            sum += vx[k];
        }
    }
    if (rows == nullptr) return;
    TO* out = rows + (size_t)blockIdx.x * width;
    if (next_w == nullptr) {
#pragma unroll
        for (int k = 0; k < VPT; ++k)
            if (threadIdx.x + k * 256 < width) out[threadIdx.x + k * 256] = from_f32<TO>(vx[k]);
        return;
    }
    mean = 0.f;
    if (next_center) mean = block_sum(sum, scratch) / (float)width;
    sq = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k)
        if (threadIdx.x + k * 256 < width) { const float v = vx[k] - mean; sq = fmaf(v, v, sq); }
    sq = block_sum(sq, scratch);
    const float next_scale = 1.0f / sqrtf(sq / (float)width + next_eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
        const int i = threadIdx.x + k * 256;
        if (i < width) out[i] = from_f32<TO>((vx[k] - mean) * next_scale * to_f32<W>(next_w[i]));
    }
}

extern "C" int qil_norm_join(void* x, int x_dtype, const float* a, const void* w, int weight_dtype, int n_rows, int width,
                             float eps, int center, const void* next_w, float next_eps, int next_center, void* rows,
                             int rows_dtype, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0) QIL_REFUSE("norm_join: width %d", width);
    if (next_w != nullptr && rows == nullptr) QIL_REFUSE("norm_join: the next norm needs rows to write");
#define QIL_JOIN_ARGS(TX, WT, TO)                                                                                   \
    dim3(n_rows), dim3(256), 0, stream, (TX*)x, a, (const WT*)w, width, eps, center, (const WT*)next_w, next_eps,   \
    next_center, (TO*)rows
#define QIL_JOIN_GO(TX, WT, TO)                                                                                     \
    do {                                                                                                            \
        if (width <= 1024) qil_launch_chained(norm_join_regs_kernel<TX, WT, TO, 4>, QIL_JOIN_ARGS(TX, WT, TO));     \
        else if (width <= 2048) qil_launch_chained(norm_join_regs_kernel<TX, WT, TO, 8>, QIL_JOIN_ARGS(TX, WT, TO)); \
        else if (width <= 4096) qil_launch_chained(norm_join_regs_kernel<TX, WT, TO, 16>, QIL_JOIN_ARGS(TX, WT, TO)); \
        else qil_launch_chained(norm_join_kernel<TX, WT, TO>, QIL_JOIN_ARGS(TX, WT, TO));                           \
    } while (0)
#define QIL_JOIN_O(TX, WT)                                                                                          \
    do { if (rows_dtype == QIL_F32) QIL_JOIN_GO(TX, WT, float); else QIL_JOIN_GO(TX, WT, bf16); } while (0)
#define QIL_JOIN_W(TX)                                                                                              \
    do { if (weight_dtype == QIL_F32) QIL_JOIN_O(TX, float); else QIL_JOIN_O(TX, bf16); } while (0)
    if (weight_dtype != QIL_F32 && weight_dtype != QIL_BF16) QIL_REFUSE("norm_join: weight dtype %d", weight_dtype);
    if (rows != nullptr && rows_dtype != QIL_F32 && rows_dtype != QIL_BF16) QIL_REFUSE("norm_join: rows dtype %d", rows_dtype);
    if (x_dtype == QIL_F32) QIL_JOIN_W(float);
    else if (x_dtype == QIL_BF16) QIL_JOIN_W(bf16);
    else QIL_REFUSE("norm_join: stream dtype %d", x_dtype);
#undef QIL_JOIN_W
#undef QIL_JOIN_O
#undef QIL_JOIN_GO
#undef QIL_JOIN_ARGS
    QIL_CHECK_LAUNCH();
}

// Several branches of one layer join the stream at once (a layer whose sublayers read the same normed row), and the
// norm of whoever reads the stream next rides along:
//   x += sum_k scale_k * b_k + sum_s y[row * top + s],   rows = norm(x; next)   (rows optional; without next.w: x rounded)
// b_k: up to four float32 branches [N, width]; a branch with a weight w_k (float32 [width]) is first divided by its root mean
// square and multiplied by it, b_k / sqrt(mean(b_k^2) + eps) * w_k.  y (optional): float32 rows of a token's `top` routed
// experts.  norm as in norm_join, or the one without statistics (below).  float32 arithmetic; every sum in the order of the
// arguments, every reduction a fixed tree over one row.
#define JOIN_MOST 4
#define JOIN_MOST_NORMED 2       // of the branches, that the register form takes
struct JoinBranches {
    const float* b[JOIN_MOST];
    const float* w[JOIN_MOST];       // null: the branch as it is
    float scale[JOIN_MOST];
    int n;
    float eps;
    const float* y;
    int top;
};
#define JOIN_RMS 0
#define JOIN_LAYER 1
#define JOIN_TANH 2
struct JoinNext {
    const void* w;       // [width]; null: no norm
    const void* b;       // [width], of w's type (JOIN_TANH)
    float eps, alpha;
    int kind;
};

template <typename T> __device__ __forceinline__ float4 join_load4(const T* p);
template <> __device__ __forceinline__ float4 join_load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 join_load4<bf16>(const bf16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void join_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void join_store4(bf16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned*>(&lo);
    raw.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
}

// Rows of up to 4 * NT * V4 values, a multiple of four, held in registers: 16 bytes a load.
template <typename TX, typename W, typename TO, int NT, int V4, bool NORMED>
__global__ void __launch_bounds__(NT)
branch_join_regs_kernel(TX* __restrict__ x, JoinBranches in, int width, JoinNext next, TO* __restrict__ rows) {
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const size_t row = blockIdx.x;
    TX* dst = x + row * width;
    float4 v[V4], stream[V4];
    float4 held[NORMED ? JOIN_MOST_NORMED : 1][NORMED ? V4 : 1];      // the normed branches' rows
    float ss[JOIN_MOST_NORMED] = {0.f, 0.f};
#pragma unroll
    for (int c = 0; c < V4; ++c) {
        const int col = (threadIdx.x + c * NT) * 4;
        v[c] = stream[c] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (NORMED) {
#pragma unroll
            for (int m = 0; m < JOIN_MOST_NORMED; ++m) held[m][c] = make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if (col >= width) continue;
        stream[c] = join_load4<TX>(dst + col);
        float4 add = make_float4(0.f, 0.f, 0.f, 0.f);
        int normed = 0;
#pragma unroll
        for (int k = 0; k < JOIN_MOST; ++k) {
            if (k >= in.n) break;
            const float4 b = *reinterpret_cast<const float4*>(in.b[k] + row * width + col);
            if (NORMED && in.w[k] != nullptr) {
#pragma unroll
                for (int m = 0; m < JOIN_MOST_NORMED; ++m)
                    if (m == normed) {
                        held[m][c] = b;
                        ss[m] = fmaf(b.x, b.x, ss[m]); ss[m] = fmaf(b.y, b.y, ss[m]);
                        ss[m] = fmaf(b.z, b.z, ss[m]); ss[m] = fmaf(b.w, b.w, ss[m]);
                    }
                ++normed;
                continue;
            }
            add.x = fmaf(in.scale[k], b.x, add.x); add.y = fmaf(in.scale[k], b.y, add.y);
            add.z = fmaf(in.scale[k], b.z, add.z); add.w = fmaf(in.scale[k], b.w, add.w);
        }
        if (in.y != nullptr)
            for (int t = 0; t < in.top; ++t) {
                const float4 b = *reinterpret_cast<const float4*>(in.y + (row * in.top + t) * width + col);
                add.x += b.x; add.y += b.y; add.z += b.z; add.w += b.w;
            }
        v[c] = add;
    }
    if (NORMED) {
        int normed = 0;
#pragma unroll
        for (int k = 0; k < JOIN_MOST; ++k) {
            if (k >= in.n) break;
            if (in.w[k] == nullptr) continue;
#pragma unroll
            for (int m = 0; m < JOIN_MOST_NORMED; ++m)
                if (m == normed) {
                    const float r = 1.0f / sqrtf(block_sum(ss[m], scratch) / (float)width + in.eps);
#pragma unroll
                    for (int c = 0; c < V4; ++c) {
                        const int col = (threadIdx.x + c * NT) * 4;
                        if (col >= width) continue;
                        const float4 w = join_load4<float>(in.w[k] + col);
                        v[c].x = fmaf(in.scale[k], held[m][c].x * r * w.x, v[c].x); v[c].y = fmaf(in.scale[k], held[m][c].y * r * w.y, v[c].y);
                        v[c].z = fmaf(in.scale[k], held[m][c].z * r * w.z, v[c].z); v[c].w = fmaf(in.scale[k], held[m][c].w * r * w.w, v[c].w);
                    }
                }
            ++normed;
        }
    }
    float sum = 0.f;
#pragma unroll
    for (int c = 0; c < V4; ++c) {
        const int col = (threadIdx.x + c * NT) * 4;
        if (col >= width) continue;
        float4 now = make_float4(stream[c].x + v[c].x, stream[c].y + v[c].y, stream[c].z + v[c].z, stream[c].w + v[c].w);
        now.x = round_to<TX>(now.x); now.y = round_to<TX>(now.y); now.z = round_to<TX>(now.z); now.w = round_to<TX>(now.w);
        join_store4(dst + col, now);
        v[c] = now;
        sum += (now.x + now.y) + (now.z + now.w);
    }
    if (rows == nullptr) return;
    TO* out = rows + row * width;
    const W* next_w = reinterpret_cast<const W*>(next.w);
    if (next_w == nullptr) {
#pragma unroll
        for (int c = 0; c < V4; ++c) {
            const int col = (threadIdx.x + c * NT) * 4;
            if (col < width) join_store4(out + col, v[c]);
        }
        return;
    }
    if (next.kind == JOIN_TANH) {
        const W* next_b = reinterpret_cast<const W*>(next.b);
#pragma unroll
        for (int c = 0; c < V4; ++c) {
            const int col = (threadIdx.x + c * NT) * 4;
            if (col >= width) continue;
            const float4 w = join_load4<W>(next_w + col), b = join_load4<W>(next_b + col);
            join_store4(out + col, make_float4(fmaf(tanhf(next.alpha * v[c].x), w.x, b.x), fmaf(tanhf(next.alpha * v[c].y), w.y, b.y),
                                               fmaf(tanhf(next.alpha * v[c].z), w.z, b.z), fmaf(tanhf(next.alpha * v[c].w), w.w, b.w)));
        }
        return;
    }
    float mean = 0.f;
    if (next.kind == JOIN_LAYER) mean = block_sum(sum, scratch) / (float)width;
    float sq = 0.f;
#pragma unroll
    for (int c = 0; c < V4; ++c) {
        if ((threadIdx.x + c * NT) * 4 >= width) continue;
        v[c].x -= mean; v[c].y -= mean; v[c].z -= mean; v[c].w -= mean;
        sq = fmaf(v[c].x, v[c].x, sq); sq = fmaf(v[c].y, v[c].y, sq);
        sq = fmaf(v[c].z, v[c].z, sq); sq = fmaf(v[c].w, v[c].w, sq);
    }
    sq = block_sum(sq, scratch);
    const float scale = 1.0f / sqrtf(sq / (float)width + next.eps);
#pragma unroll
    for (int c = 0; c < V4; ++c) {
        const int col = (threadIdx.x + c * NT) * 4;
        if (col >= width) continue;
        const float4 w = join_load4<W>(next_w + col);
        join_store4(out + col, make_float4(v[c].x * scale * w.x, v[c].y * scale * w.y, v[c].z * scale * w.z, v[c].w * scale * w.w));
    }
}

// Any width and number of normed branches: the stream's row is read back by the threads that wrote it.
template <typename TX, typename W, typename TO>
__global__ void __launch_bounds__(256)
branch_join_kernel(TX* __restrict__ x, JoinBranches in, int width, JoinNext next, TO* __restrict__ rows) {
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const size_t row = blockIdx.x;
    TX* dst = x + row * width;
    float r[JOIN_MOST];
#pragma unroll
    for (int k = 0; k < JOIN_MOST; ++k) {
        r[k] = 1.f;
        if (k >= in.n || in.w[k] == nullptr) continue;
        float ss = 0.f;
        for (int i = threadIdx.x; i < width; i += 256) { const float v = in.b[k][row * width + i]; ss = fmaf(v, v, ss); }
        r[k] = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + in.eps);
    }
    float sum = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        float add = 0.f;
#pragma unroll
        for (int k = 0; k < JOIN_MOST; ++k)
            if (k < in.n && in.w[k] == nullptr) add = fmaf(in.scale[k], in.b[k][row * width + i], add);
        if (in.y != nullptr)
            for (int t = 0; t < in.top; ++t) add += in.y[(row * in.top + t) * width + i];
#pragma unroll
        for (int k = 0; k < JOIN_MOST; ++k)
            if (k < in.n && in.w[k] != nullptr) add = fmaf(in.scale[k], in.b[k][row * width + i] * r[k] * in.w[k][i], add);
        const TX now = from_f32<TX>(to_f32<TX>(dst[i]) + add);
        dst[i] = now;
        sum += to_f32<TX>(now);
    }
    if (rows == nullptr) return;
    TO* out = rows + row * width;
    const W* next_w = reinterpret_cast<const W*>(next.w);
    if (next_w == nullptr) {
        for (int i = threadIdx.x; i < width; i += 256) out[i] = from_f32<TO>(to_f32<TX>(dst[i]));
        return;
    }
    if (next.kind == JOIN_TANH) {
        const W* next_b = reinterpret_cast<const W*>(next.b);
        for (int i = threadIdx.x; i < width; i += 256)
            out[i] = from_f32<TO>(fmaf(tanhf(next.alpha * to_f32<TX>(dst[i])), to_f32<W>(next_w[i]), to_f32<W>(next_b[i])));
        return;
    }
    float mean = 0.f;
    if (next.kind == JOIN_LAYER) mean = block_sum(sum, scratch) / (float)width;
    float sq = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) {
        const float v = to_f32<TX>(dst[i]) - mean;
        sq = fmaf(v, v, sq);
    }
    sq = block_sum(sq, scratch);
    const float scale = 1.0f / sqrtf(sq / (float)width + next.eps);
    for (int i = threadIdx.x; i < width; i += 256)
        out[i] = from_f32<TO>((to_f32<TX>(dst[i]) - mean) * scale * to_f32<W>(next_w[i]));
}

// branches, weights (entries may be null): host arrays of n device pointers; scales: host array of n.
extern "C" int qil_branch_join(void* x, int x_dtype, const float* const* branches, const float* const* weights, const float* scales,
                               int n_branches, float branch_eps, const float* y, int top, int n_rows, int width,
                               const void* next_w, const void* next_b, int weight_dtype, float next_eps, float next_alpha,
                               int next_kind, void* rows, int rows_dtype, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0 || n_branches < 0 || n_branches > JOIN_MOST || (y != nullptr && top < 1))
        QIL_REFUSE("branch_join: width %d, %d branches (at most %d), %d experts a token", width, n_branches, JOIN_MOST, top);
    if (next_w != nullptr && rows == nullptr) QIL_REFUSE("branch_join: the next norm needs rows to write");
    if (next_kind < 0 || next_kind > JOIN_TANH || (next_w != nullptr && next_kind == JOIN_TANH && next_b == nullptr))
        QIL_REFUSE("branch_join: next norm %d", next_kind);
    JoinBranches in = {};
    uintptr_t bits = (uintptr_t)x | (uintptr_t)y | (uintptr_t)next_w | (uintptr_t)next_b | (uintptr_t)rows;
    int normed = 0;
    for (int k = 0; k < n_branches; ++k) {
        in.b[k] = branches[k]; in.scale[k] = scales[k]; in.w[k] = weights != nullptr ? weights[k] : nullptr;
        bits |= (uintptr_t)branches[k] | (uintptr_t)in.w[k];
        if (in.w[k] != nullptr) ++normed;
    }
    in.n = n_branches; in.eps = branch_eps; in.y = y; in.top = top;
    const JoinNext next = {next_w, next_b, next_eps, next_alpha, next_kind};
    const bool wide = width % 4 == 0 && (bits & 15) == 0 && normed <= JOIN_MOST_NORMED;
#define QIL_JOIN_ARGS(TX, TO, NT) dim3(n_rows), dim3(NT), 0, stream, (TX*)x, in, width, next, (TO*)rows
#define QIL_JOIN_SIZE(TX, WT, TO, N)                                                                                           \
    do {                                                                                                                       \
        if (width <= 1024) qil_launch_chained(branch_join_regs_kernel<TX, WT, TO, 256, 1, N>, QIL_JOIN_ARGS(TX, TO, 256));     \
        else if (width <= 2048) qil_launch_chained(branch_join_regs_kernel<TX, WT, TO, 256, 2, N>, QIL_JOIN_ARGS(TX, TO, 256)); \
        else qil_launch_chained(branch_join_regs_kernel<TX, WT, TO, 512, 2, N>, QIL_JOIN_ARGS(TX, TO, 512));                   \
    } while (0)
#define QIL_JOIN_GO(TX, WT, TO)                                                                                                \
    do {                                                                                                                       \
        if (!wide || width > 4096) qil_launch_chained(branch_join_kernel<TX, WT, TO>, QIL_JOIN_ARGS(TX, TO, 256));                  \
        else if (normed) QIL_JOIN_SIZE(TX, WT, TO, true);                                                                      \
        else QIL_JOIN_SIZE(TX, WT, TO, false);                                                                                 \
    } while (0)
#define QIL_JOIN_O(TX, WT)                                                                                            \
    do { if (rows_dtype == QIL_F32) QIL_JOIN_GO(TX, WT, float); else QIL_JOIN_GO(TX, WT, bf16); } while (0)
#define QIL_JOIN_W(TX)                                                                                                \
    do { if (weight_dtype == QIL_F32) QIL_JOIN_O(TX, float); else QIL_JOIN_O(TX, bf16); } while (0)
    if (next_w != nullptr && weight_dtype != QIL_F32 && weight_dtype != QIL_BF16) QIL_REFUSE("branch_join: weight dtype %d", weight_dtype);
    if (rows != nullptr && rows_dtype != QIL_F32 && rows_dtype != QIL_BF16) QIL_REFUSE("branch_join: rows dtype %d", rows_dtype);
    if (x_dtype == QIL_F32) QIL_JOIN_W(float);
    else if (x_dtype == QIL_BF16) QIL_JOIN_W(bf16);
    else QIL_REFUSE("branch_join: stream dtype %d", x_dtype);
#undef QIL_JOIN_W
#undef QIL_JOIN_O
#undef QIL_JOIN_GO
#undef QIL_JOIN_SIZE
#undef QIL_JOIN_ARGS
    QIL_CHECK_LAUNCH();
}

// The norm without statistics (Dynamic Tanh): y = tanh(alpha x) * w + b, float32 arithmetic, one rounding.
template <typename TI, typename TO, typename W>
__global__ void __launch_bounds__(256)
tanh_norm_kernel(const TI* __restrict__ x, const W* __restrict__ weight, const W* __restrict__ bias, float alpha,
                 const int* __restrict__ rows, TO* __restrict__ out, int width) {
    qil_wait_for_producer();
    qil_release_consumer();
    const int r = blockIdx.x;
    const TI* src = x + (size_t)(rows ? rows[r] : r) * width;
    TO* dst = out + (size_t)r * width;
    for (int i = threadIdx.x; i < width; i += 256)
        dst[i] = from_f32<TO>(fmaf(tanhf(alpha * to_f32<TI>(src[i])), to_f32<W>(weight[i]), to_f32<W>(bias[i])));
}

extern "C" int qil_tanh_norm(const void* x, int x_dtype, const void* weight, const void* bias, int weight_dtype, float alpha,
                             const int* rows, void* out, int out_dtype, int n_rows, int width, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0) QIL_REFUSE("tanh_norm: width %d", width);
    if (weight_dtype != QIL_F32 && weight_dtype != QIL_BF16) QIL_REFUSE("tanh_norm: weight dtype %d", weight_dtype);
#define QIL_TANH_GO(TI, TO)                                                                                                  \
    do {                                                                                                                     \
        if (weight_dtype == QIL_F32)                                                                                         \
            qil_launch_chained(tanh_norm_kernel<TI, TO, float>, dim3(n_rows), dim3(256), 0, stream, (const TI*)x,            \
                               (const float*)weight, (const float*)bias, alpha, rows, (TO*)out, width);                      \
        else                                                                                                                 \
            qil_launch_chained(tanh_norm_kernel<TI, TO, bf16>, dim3(n_rows), dim3(256), 0, stream, (const TI*)x,             \
                               (const bf16*)weight, (const bf16*)bias, alpha, rows, (TO*)out, width);                        \
    } while (0)
    if (x_dtype == QIL_F32 && out_dtype == QIL_F32) QIL_TANH_GO(float, float);
    else if (x_dtype == QIL_F32 && out_dtype == QIL_BF16) QIL_TANH_GO(float, bf16);
    else if (x_dtype == QIL_BF16 && out_dtype == QIL_BF16) QIL_TANH_GO(bf16, bf16);
    else if (x_dtype == QIL_BF16 && out_dtype == QIL_F32) QIL_TANH_GO(bf16, float);
    else QIL_REFUSE("tanh_norm: dtypes %d -> %d", x_dtype, out_dtype);
#undef QIL_TANH_GO
    QIL_CHECK_LAUNCH();
}

// Memory-bound row kernels: embedding gather, RMSNorm (optionally through a row
// index), SiLU-gate multiply, in-place add and dtype casts.
//
// Formulas follow the reference: the norm squares, averages, adds eps, takes the
// reciprocal square root and scales in float32, rounds to the activation dtype and
// only then multiplies by the weight (qil/model.py:21-23); the gate is
// silu(gate) rounded to the activation dtype, times up (qil/model.py:71).
#include "common.cuh"

QIL_ERROR_STORAGE

// ---------------------------------------------------------------- embedding
template <typename T, typename W>
__global__ void embed_gather_kernel(const W* __restrict__ table, const int* __restrict__ ids,
                                    T* __restrict__ out, int width, int vocab, float scale,
                                    const W* __restrict__ pos_table, const int* __restrict__ positions, int n_positions) {
    const int row = blockIdx.x;
    int id = ids[row];
    // Host code validates ids; clamp so that a bad id can never read out of bounds.
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    const W* src = table + (size_t)id * width;
    T* dst = out + (size_t)row * width;
    if (pos_table != nullptr) {
        int p = positions[row];
        p = p < 0 ? 0 : (p >= n_positions ? n_positions - 1 : p);
        const W* at = pos_table + (size_t)p * width;
        for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = from_f32<T>(to_f32<W>(src[i]) * scale + to_f32<W>(at[i]));
        return;
    }
    for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = from_f32<T>(to_f32<W>(src[i]) * scale);
}

// bfloat16 table and output with a width that allows 16-byte copies
__global__ void embed_gather_bf16x8_kernel(const bf16* __restrict__ table, const int* __restrict__ ids,
                                           bf16* __restrict__ out, int width, int vocab) {
    qil_wait_for_producer();
    qil_release_consumer();
    const int row = blockIdx.x;
    int id = ids[row];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    const uint4* src = reinterpret_cast<const uint4*>(table + (size_t)id * width);
    uint4* dst = reinterpret_cast<uint4*>(out + (size_t)row * width);
    for (int i = threadIdx.x; i < width / 8; i += blockDim.x) dst[i] = src[i];
}

extern "C" int qil_embed_gather(const void* table, int table_dtype, const int* ids, void* out,
                                int out_dtype, int n_rows, int width, int vocab, float scale, const void* pos_table,
                                const int* positions, int n_positions, cudaStream_t stream) {
    // scale: what every row is multiplied by on its way out (float32 product, one rounding).  pos_table (null: none), of
    // the table's type, [n_positions, width]: the row of the token's position is added, unscaled, before the rounding
    if (n_rows <= 0) return 0;
    if (width <= 0 || vocab <= 0) QIL_REFUSE("embed_gather: width %d vocab %d", width, vocab);
    if (pos_table != nullptr && (positions == nullptr || n_positions <= 0))
        QIL_REFUSE("embed_gather: a table of %d positions", n_positions);
    if (pos_table == nullptr && scale == 1.0f && out_dtype == QIL_BF16 && table_dtype == QIL_BF16 && width % 8 == 0 &&
        (((uintptr_t)table | (uintptr_t)out) & 15) == 0) {
        qil_launch_chained(embed_gather_bf16x8_kernel, dim3(n_rows), dim3(128), 0, stream,
                           (const bf16*)table, ids, (bf16*)out, width, vocab);
        QIL_CHECK_LAUNCH();
    }
    QIL_DISPATCH_2(out_dtype, table_dtype,
        embed_gather_kernel<T, W><<<n_rows, 256, 0, stream>>>((const W*)table, ids, (T*)out, width, vocab, scale,
                                                        (const W*)pos_table, positions, n_positions));
    QIL_CHECK_LAUNCH();
}

// ---------------------------------------------------------------- RMSNorm
// One block per output row.  rows == nullptr: row r reads x[r]; else x[rows[r]].
template <typename T, typename W>
__global__ void rmsnorm_kernel(const T* __restrict__ x, const W* __restrict__ weight,
                               const int* __restrict__ rows, T* __restrict__ out,
                               int width, float eps) {
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    const int src_row = rows ? rows[r] : r;
    const T* src = x + (size_t)src_row * width;
    T* dst = out + (size_t)r * width;
    float sq = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = to_f32<T>(src[i]);
        sq += v * v;
    }
    sq = block_sum(sq, scratch);
    const float scale = 1.0f / sqrtf(sq / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float normed = round_to<T>(to_f32<T>(src[i]) * scale);
        dst[i] = from_f32<T>(normed * to_f32<W>(weight[i]));
    }
}

// bfloat16 rows of up to 256 * 8 * RMS_VPT elements: the whole row sits in registers, every load is
// 16 bytes wide and issued before the first use, so a row costs one memory round trip, not one per element.
#define RMS_VPT 4
template <typename W>
__global__ void __launch_bounds__(256)
rmsnorm_bf16x8_kernel(const bf16* __restrict__ x, const W* __restrict__ weight, const int* __restrict__ rows,
                      bf16* __restrict__ out, int width, float eps) {
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const int r = blockIdx.x;
    const int src_row = rows ? rows[r] : r;
    const uint4* src = reinterpret_cast<const uint4*>(x + (size_t)src_row * width);
    uint4* dst = reinterpret_cast<uint4*>(out + (size_t)r * width);
    const int vectors = width / 8;
    uint4 v[RMS_VPT];
#pragma unroll
    for (int i = 0; i < RMS_VPT; ++i) {
        const int idx = threadIdx.x + i * 256;
        v[i] = idx < vectors ? src[idx] : make_uint4(0u, 0u, 0u, 0u);
    }
    float sq = 0.f;
#pragma unroll
    for (int i = 0; i < RMS_VPT; ++i) {
        const bf16* e = reinterpret_cast<const bf16*>(&v[i]);
#pragma unroll
        for (int k = 0; k < 8; ++k) { const float f = __bfloat162float(e[k]); sq += f * f; }
    }
    sq = block_sum(sq, scratch);
    const float scale = 1.0f / sqrtf(sq / (float)width + eps);
#pragma unroll
    for (int i = 0; i < RMS_VPT; ++i) {
        const int idx = threadIdx.x + i * 256;
        if (idx >= vectors) continue;
        uint4 o4;
        if (sizeof(W) == 2) {
            // bfloat16 weights: one 16-byte read, and the product of the rounded value and the weight as a
            // packed bfloat16 multiply (one rounding, never contracted with anything)
            const uint4 w4 = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(weight) + idx * 8);
            const __nv_bfloat162* e2 = reinterpret_cast<const __nv_bfloat162*>(&v[i]);
            const __nv_bfloat162* w2 = reinterpret_cast<const __nv_bfloat162*>(&w4);
            __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&o4);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 f = __bfloat1622float2(e2[k]);
                o2[k] = __hmul2_rn(__floats2bfloat162_rn(f.x * scale, f.y * scale), w2[k]);
            }
        } else {
            const bf16* e = reinterpret_cast<const bf16*>(&v[i]);
            bf16* o = reinterpret_cast<bf16*>(&o4);
#pragma unroll
            for (int k = 0; k < 8; ++k) {
                const float normed = round_to<bf16>(__bfloat162float(e[k]) * scale);
                o[k] = __float2bfloat16_rn(normed * to_f32<W>(weight[idx * 8 + k]));
            }
        }
        dst[idx] = o4;
    }
}

extern "C" int qil_rmsnorm(const void* x, const void* weight, const int* rows, void* out,
                           int n_rows, int width, float eps, int act_dtype, int weight_dtype,
                           cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0) QIL_REFUSE("rmsnorm: width %d", width);
    if (act_dtype == QIL_BF16 && width % 8 == 0 && width <= 256 * 8 * RMS_VPT &&
        (((uintptr_t)x | (uintptr_t)out | (uintptr_t)weight) & 15) == 0) {
        if (weight_dtype == QIL_BF16)
            qil_launch_chained(rmsnorm_bf16x8_kernel<bf16>, dim3(n_rows), dim3(256), 0, stream,
                               (const bf16*)x, (const bf16*)weight, rows, (bf16*)out, width, eps);
        else if (weight_dtype == QIL_F32)
            qil_launch_chained(rmsnorm_bf16x8_kernel<float>, dim3(n_rows), dim3(256), 0, stream,
                               (const bf16*)x, (const float*)weight, rows, (bf16*)out, width, eps);
        else QIL_REFUSE("unknown dtype code %d", weight_dtype);
        QIL_CHECK_LAUNCH();
    }
    QIL_DISPATCH_2(act_dtype, weight_dtype,
        rmsnorm_kernel<T, W><<<n_rows, 256, 0, stream>>>((const T*)x, (const W*)weight, rows, (T*)out, width, eps));
    QIL_CHECK_LAUNCH();
}

// ---------------------------------------------------------------- SiLU(gate) * up
// gate_up: [n_rows, 2 * width]; out: [n_rows, width].  pairs8 == 0: gate columns first, then up
// columns.  pairs8 == 1: groups of 16 columns, 8 gate columns then the 8 matching up columns
// (the layout the decode GEMM's fused epilogue wants its weight rows in).
template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ gate_up, T* __restrict__ out, int width,
                                size_t total, int pairs8) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; i < total; i += stride) {
        const size_t row = i / width;
        const int col = (int)(i - row * width);
        const int gcol = pairs8 ? (col >> 3) * 16 + (col & 7) : col;
        const int ucol = pairs8 ? gcol + 8 : width + col;
        const float g = to_f32<T>(gate_up[row * 2 * width + gcol]);
        const float u = to_f32<T>(gate_up[row * 2 * width + ucol]);
        const float act = round_to<T>(g / (1.0f + expf(-g)));
        out[i] = from_f32<T>(act * u);
    }
}

// 8 bf16 values per thread when the width allows 16-byte accesses.
__global__ void silu_mul_bf16x8_kernel(const bf16* __restrict__ gate_up, bf16* __restrict__ out,
                                       int width, size_t total_vec, int pairs8) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    const int vec_per_row = width / 8;
    for (; i < total_vec; i += stride) {
        const size_t row = i / vec_per_row;
        const int col = (int)(i - row * vec_per_row) * 8;
        const int gcol = pairs8 ? 2 * col : col;
        const int ucol = pairs8 ? 2 * col + 8 : width + col;
        const uint4 g4 = *reinterpret_cast<const uint4*>(gate_up + row * 2 * width + gcol);
        const uint4 u4 = *reinterpret_cast<const uint4*>(gate_up + row * 2 * width + ucol);
        const bf16* g = reinterpret_cast<const bf16*>(&g4);
        const bf16* u = reinterpret_cast<const bf16*>(&u4);
        uint4 o4;
        bf16* o = reinterpret_cast<bf16*>(&o4);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            const float gv = __bfloat162float(g[k]);
            // fast exp and divide (a few ulp in float32): the value is rounded to bfloat16 next
            const float act = round_to<bf16>(__fdividef(gv, 1.0f + __expf(-gv)));
            o[k] = __float2bfloat16_rn(act * __bfloat162float(u[k]));
        }
        *reinterpret_cast<uint4*>(out + row * width + col) = o4;
    }
}

extern "C" int qil_silu_mul(const void* gate_up, void* out, int n_rows, int width, int act_dtype,
                            int pairs8, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0) QIL_REFUSE("silu_mul: width %d", width);
    if (pairs8 && width % 8) QIL_REFUSE("silu_mul: the paired layout needs a width that is a multiple of 8, got %d", width);
    const size_t total = (size_t)n_rows * width;
    if (act_dtype == QIL_BF16 && width % 8 == 0 && ((uintptr_t)gate_up % 16) == 0 && ((uintptr_t)out % 16) == 0) {
        const size_t total_vec = total / 8;
        const int blocks = (int)((total_vec + 255) / 256 < 148 * 16 ? (total_vec + 255) / 256 : 148 * 16);
        silu_mul_bf16x8_kernel<<<blocks, 256, 0, stream>>>((const bf16*)gate_up, (bf16*)out, width, total_vec, pairs8);
        QIL_CHECK_LAUNCH();
    }
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    QIL_DISPATCH_1(act_dtype,
        silu_mul_kernel<T><<<blocks, 256, 0, stream>>>((const T*)gate_up, (T*)out, width, total, pairs8));
    QIL_CHECK_LAUNCH();
}

// ---------------------------------------------------------------- x += y (float32 sum, one rounding)
template <typename T>
__global__ void add_inplace_kernel(T* __restrict__ x, const T* __restrict__ y, size_t total) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; i < total; i += stride) x[i] = from_f32<T>(to_f32<T>(x[i]) + to_f32<T>(y[i]));
}

extern "C" int qil_add_inplace(void* x, const void* y, long long total, int act_dtype, cudaStream_t stream) {
    if (total <= 0) return 0;
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    QIL_DISPATCH_1(act_dtype,
        add_inplace_kernel<T><<<blocks, 256, 0, stream>>>((T*)x, (const T*)y, (size_t)total));
    QIL_CHECK_LAUNCH();
}


// ---------------------------------------------------------------- scaled add
// x[r][c] += scale[c] * y[r][c]: a branch joins the residual stream through a learned scale per feature.
// float32 arithmetic; x and y may differ in type (a float32 stream, bfloat16 branch).
template <typename TX, typename TY>
__global__ void __launch_bounds__(256)
scaled_add_kernel(TX* __restrict__ x, const TY* __restrict__ y, const float* __restrict__ scale, int n_rows, int width) {
    qil_wait_for_producer();
    qil_release_consumer();
    // a block walks rows, a thread the same columns of each: no division per element, the scale read once
    for (int col = threadIdx.x; col < width; col += 256) {
        const float s = scale[col];
        for (int row = blockIdx.x; row < n_rows; row += gridDim.x) {
            const size_t i = (size_t)row * width + col;
            x[i] = from_f32<TX>(fmaf(s, to_f32<TY>(y[i]), to_f32<TX>(x[i])));
        }
    }
}

// float32 stream, widths that are multiples of 4: 16 bytes a load
template <typename TY>
__global__ void __launch_bounds__(256)
scaled_add_f32x4_kernel(float* __restrict__ x, const TY* __restrict__ y, const float* __restrict__ scale, int n_rows, int width) {
    qil_wait_for_producer();
    qil_release_consumer();
    for (int col = threadIdx.x * 4; col < width; col += 1024) {
        const float4 s = *reinterpret_cast<const float4*>(scale + col);
        for (int row = blockIdx.x; row < n_rows; row += gridDim.x) {
            const size_t i = (size_t)row * width + col;
            float4 v = *reinterpret_cast<float4*>(x + i);
            float b[4];
            if (sizeof(TY) == 4) {
                const float4 t = *reinterpret_cast<const float4*>(y + i);
                b[0] = t.x; b[1] = t.y; b[2] = t.z; b[3] = t.w;
            } else {
                const uint2 raw = *reinterpret_cast<const uint2*>(y + i);
                const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
                const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
                b[0] = lo.x; b[1] = lo.y; b[2] = hi.x; b[3] = hi.y;
            }
            v.x = fmaf(s.x, b[0], v.x); v.y = fmaf(s.y, b[1], v.y); v.z = fmaf(s.z, b[2], v.z); v.w = fmaf(s.w, b[3], v.w);
            *reinterpret_cast<float4*>(x + i) = v;
        }
    }
}

extern "C" int qil_scaled_add(void* x, int x_dtype, const void* y, int y_dtype, const float* scale, int n_rows,
                              int width, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0) QIL_REFUSE("scaled_add: width %d", width);
    const int blocks = n_rows < 148 * 8 ? n_rows : 148 * 8;
    if (x_dtype == QIL_F32 && width % 4 == 0 && (((uintptr_t)x | (uintptr_t)y | (uintptr_t)scale) & 15) == 0) {
        if (y_dtype == QIL_F32)
            qil_launch_chained(scaled_add_f32x4_kernel<float>, dim3(blocks), dim3(256), 0, stream, (float*)x, (const float*)y, scale, n_rows, width);
        else if (y_dtype == QIL_BF16)
            qil_launch_chained(scaled_add_f32x4_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (float*)x, (const bf16*)y, scale, n_rows, width);
        else QIL_REFUSE("scaled_add: dtypes %d += %d", x_dtype, y_dtype);
        QIL_CHECK_LAUNCH();
    }
#define QIL_GO(TX, TY) qil_launch_chained(scaled_add_kernel<TX, TY>, dim3(blocks), dim3(256), 0, stream, (TX*)x, (const TY*)y, scale, n_rows, width)
    if (x_dtype == QIL_F32 && y_dtype == QIL_F32) QIL_GO(float, float);
    else if (x_dtype == QIL_F32 && y_dtype == QIL_BF16) QIL_GO(float, bf16);
    else if (x_dtype == QIL_BF16 && y_dtype == QIL_BF16) QIL_GO(bf16, bf16);
    else if (x_dtype == QIL_BF16 && y_dtype == QIL_F32) QIL_GO(bf16, float);
    else QIL_REFUSE("scaled_add: dtypes %d += %d", x_dtype, y_dtype);
#undef QIL_GO
    QIL_CHECK_LAUNCH();
}
// ---------------------------------------------------------------- token ids that are still on the device
// token_ids[pairs[2i]] = source[pairs[2i + 1]]: a step may be queued before the host has read the tokens
// that the step before it sampled; their places in the step's token list are filled in here, on the
// stream, from the sampler's device buffer.  A source index outside [0, n_source) leaves the place as it is.
__global__ void feed_tokens_kernel(int* __restrict__ token_ids, const int* __restrict__ pairs, int count,
                                   const int* __restrict__ source, int n_source, int n_tokens) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= count) return;
    const int dst = pairs[2 * i], src = pairs[2 * i + 1];
    if (dst >= 0 && dst < n_tokens && src >= 0 && src < n_source) token_ids[dst] = source[src];
}

extern "C" int qil_feed_tokens(int* token_ids, const int* pairs, int count, const int* source, int n_source,
                               int n_tokens, cudaStream_t stream) {
    if (count <= 0) return 0;
    feed_tokens_kernel<<<(count + 127) / 128, 128, 0, stream>>>(token_ids, pairs, count, source, n_source, n_tokens);
    QIL_CHECK_LAUNCH();
}

// ---------------------------------------------------------------- dtype cast (src dtype -> dst dtype)
template <typename T, typename W>
__global__ void cast_kernel(const W* __restrict__ src, T* __restrict__ dst, size_t total) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; i < total; i += stride) dst[i] = from_f32<T>(to_f32<W>(src[i]));
}

extern "C" int qil_cast(const void* src, int src_dtype, void* dst, int dst_dtype, long long total,
                        cudaStream_t stream) {
    if (total <= 0) return 0;
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    QIL_DISPATCH_2(dst_dtype, src_dtype,
        cast_kernel<T, W><<<blocks, 256, 0, stream>>>((const W*)src, (T*)dst, (size_t)total));
    QIL_CHECK_LAUNCH();
}

// ---------------------------------------------------------------- random weights
// out[i] = mean + std * z(seed, i) with z close to N(0, 1): the sum of twelve 16-bit uniforms drawn from
// three rounds of a 64-bit counter hash, centred and divided by 65536.  Integer arithmetic and three
// correctly rounded float operations only, so the host twin (weights/random_init.py) gives the same bits.
__device__ __forceinline__ unsigned long long fill_hash(unsigned long long seed, unsigned long long counter) {
    unsigned long long z = seed + (counter + 1ull) * 0x9E3779B97F4A7C15ull;
    z ^= z >> 30; z *= 0xBF58476D1CE4E5B9ull;
    z ^= z >> 27; z *= 0x94D049BB133111EBull;
    z ^= z >> 31;
    return z;
}

template <typename T>
__global__ void fill_normal_kernel(T* __restrict__ out, long long total, unsigned long long seed, float std,
                                   float mean) {
    const long long stride = (long long)gridDim.x * blockDim.x;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) {
        int sum = 0;
#pragma unroll
        for (int round = 0; round < 3; ++round) {
            const unsigned long long h = fill_hash(seed, 3ull * (unsigned long long)i + round);
            sum += (int)(h & 0xFFFFull) + (int)((h >> 16) & 0xFFFFull) + (int)((h >> 32) & 0xFFFFull) + (int)(h >> 48);
        }
        const float z = __fmul_rn((float)(sum - 393210), 1.0f / 65536.0f);
        out[i] = from_f32<T>(__fadd_rn(__fmul_rn(z, std), mean));
    }
}

extern "C" int qil_fill_normal(void* out, int out_dtype, long long total, unsigned long long seed, float std,
                               float mean, cudaStream_t stream) {
    if (total <= 0) return 0;
    const long long blocks = (total + 255) / 256;
    const int grid = (int)(blocks < 148 * 16 ? blocks : 148 * 16);
    QIL_DISPATCH_1(out_dtype, fill_normal_kernel<T><<<grid, 256, 0, stream>>>((T*)out, total, seed, std, mean));
    QIL_CHECK_LAUNCH();
}

// ---------------------------------------------------------------- x *= s (float32 rows, e.g. logits)
__global__ void scale_inplace_kernel(float* __restrict__ x, size_t total, float s) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; i < total; i += stride) x[i] *= s;
}

// x <- cap * tanh(x / cap) (float32 rows, e.g. logits)
__global__ void softcap_inplace_kernel(float* __restrict__ x, size_t total, float cap) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    for (; i < total; i += stride) x[i] = cap * tanhf(x[i] / cap);
}

extern "C" int qil_softcap_inplace(float* x, long long total, float cap, cudaStream_t stream) {
    if (total <= 0) return 0;
    if (!(cap > 0.f)) QIL_REFUSE("softcap_inplace: a cap of %g", (double)cap);
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    softcap_inplace_kernel<<<blocks, 256, 0, stream>>>(x, (size_t)total, cap);
    QIL_CHECK_LAUNCH();
}

extern "C" int qil_scale_inplace(float* x, long long total, float s, cudaStream_t stream) {
    if (total <= 0) return 0;
    const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
    scale_inplace_kernel<<<blocks, 256, 0, stream>>>(x, (size_t)total, s);
    QIL_CHECK_LAUNCH();
}

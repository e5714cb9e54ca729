// Recurrences with a state matrix S [d, e] per head (float32, one per request) and one decay g per token and head, with or
// without the delta rule's correction:
//
//   plain:   S <- g S + k v^T                                                    o = S^T q
//   delta:   S <- g S,   u = beta (v - S^T k),   S <- S + k u^T                  o = S^T q
//
// q and k come as float32 rows that other kernels made (unit vectors, rotated, scaled: whatever enters the recurrence), one
// q/k head for every `group` heads; v as columns of a row-major buffer in the activations' type.  The decay is a fixed number
// per head (`head_decay`) or a logarithm per token and head (`log_decay`).  Everything from there on is float32.
//
// Two forms.  state_scan walks a segment token by token from the request's slot (single tokens, short portions): its result
// does not depend on the cut to the last bit.  Long portions are cut into chunks of MS_CHUNK tokens (beginning where the
// portion begins) and take matrix products instead of a walk.  With L_i the sum of the log decays of a chunk up to token i, S
// the state that comes into the chunk, and k_i, v_i, q_i, beta_i as above, the correction makes u a triangular system:
//
//   u_i + sum_{j < i} beta_i e^(L_i - L_j) (k_i . k_j) u_j  =  beta_i v_i - beta_i e^(L_i) S^T k_i
//
// so with A the strictly lower matrix of those coefficients, U = (I + A)^-1 diag(beta) V and
// W = (I + A)^-1 diag(beta e^L) K (delta_solve, all chunks at once: an explicit inverse by blocks),
//
//   Y = U - W S            (plain: Y = V)                                    delta_walk: the chunks of a portion in order,
//   S' = e^(L_C) S + sum_j e^(L_C - L_j) k_j y_j^T                           a block per (head, a few value columns)
//   o_i = e^(L_i) S^T q_i + sum_{j <= i} e^(L_i - L_j) (q_i . k_j) y_j       state_outputs: all chunks at once
//
// Without the correction the sums of S' need no S: state_own makes them for all chunks at once and gla_carry walks them.
// Every exponential is of a difference of sums kept in double precision and is at most one.  Chunks round differently from
// the walk by token, in the last bits.
#include "common.cuh"
#include "head_norm_gate.cuh"

#define MS_CHUNK 64
#define MS_MOST_D 256        // key channels of a head that the chunked form holds in shared memory

struct StateRows {
    const float* q;              // float32 [tokens, qk_ld]: head g's q at column g * d
    const float* k;
    long long qk_ld;
    int group;                   // heads per q/k head
    const void* v;               // T: head h's values at column h * e
    long long v_ld;
    const float* log_decay;      // float32 [tokens, heads], or null
    const float* head_decay;     // float32 [heads], or null
    const float* beta;           // float32 [tokens, heads] (delta)
};

// ------------------------------------------------------------------ token by token
#define MS_R 32              // rows of a column that one thread holds
#define MS_TB 8              // tokens staged at a time
#define MS_THREADS 512

// A thread holds MS_R rows of one value column; ds_count threads (a power of two within a warp) share the column.  With the
// correction, S^T k and S^T q are taken from the state as it stands (one pass, one reduction): with sk, sq those sums,
// u = beta (v - g sk), o = g sq + (k . q) u, and the state moves on.  NORM: the block holds all of a head's columns and
// norms and gates its outputs itself.
template <typename T, bool DELTA, bool NORM>
__global__ void __launch_bounds__(MS_THREADS, 1)
state_scan_kernel(StateRows in, const T* __restrict__ gate, long long gate_ld, const float* __restrict__ norm_w, float eps,
                  float* __restrict__ state, const int* __restrict__ seg_start, const int* __restrict__ seg_len,
                  const int* __restrict__ seg_row, int n_heads, int d, int e, int ds_count, int tile_cols,
                  float* __restrict__ o_raw, T* __restrict__ out) {
    extern __shared__ __align__(16) float smem[];
    // a token's q and k: ds_count blocks of MS_R values, each followed by four unused floats (bank spread)
    const int stride = ds_count * (MS_R + 4);
    float* sq = smem;                       // [TB][stride]
    float* sk = sq + MS_TB * stride;        // [TB][stride]
    float* sv = sk + MS_TB * stride;        // [TB][tile_cols]
    float* so = sv + MS_TB * tile_cols;     // [TB][tile_cols]
    float* sg = so + MS_TB * tile_cols;     // [TB] decays
    float* sb = sg + MS_TB;                 // [TB] betas
    float* skq = sb + MS_TB;                // [TB] k . q
    const int tiles = (e + tile_cols - 1) / tile_cols;
    const int head = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * tile_cols, seg = blockIdx.y;
    const int first = seg_start[seg], count = seg_len[seg], row = seg_row[seg];      // the step's description: uploaded before
    const int tid = threadIdx.x, threads = blockDim.x, lane = tid & 31, warp = tid >> 5, warps = threads >> 5;
    const int local = tid / ds_count, ds = tid % ds_count;
    const bool owner = local < tile_cols && col0 + local < e;
    const size_t qk_at = (size_t)(head / in.group) * d;
    const T* v = reinterpret_cast<const T*>(in.v);
    float* slot = state + ((size_t)row * n_heads + head) * d * e + (size_t)ds * MS_R * e + col0 + local;
    qil_wait_for_producer();
    qil_release_consumer();
    float S[MS_R];
#pragma unroll
    for (int r = 0; r < MS_R; ++r) S[r] = (owner && ds * MS_R + r < d) ? slot[(size_t)r * e] : 0.f;
    for (int t0 = 0; t0 < count; t0 += MS_TB) {
        const int nb = count - t0 < MS_TB ? count - t0 : MS_TB;
        __syncthreads();
        for (int i = tid; i < nb * ds_count * MS_R; i += threads) {
            const int tb = i / (ds_count * MS_R), dd = i % (ds_count * MS_R);
            const int to = tb * stride + (dd / MS_R) * (MS_R + 4) + dd % MS_R;
            const size_t from = (size_t)(first + t0 + tb) * in.qk_ld + qk_at + dd;
            sq[to] = dd < d ? in.q[from] : 0.f;          // rows past d: zeros, which keep their (zero) state rows zero
            sk[to] = dd < d ? in.k[from] : 0.f;
        }
        for (int i = tid; i < nb * tile_cols; i += threads) {
            const int tb = i / tile_cols, c = col0 + i % tile_cols;
            sv[i] = c < e ? to_f32<T>(v[(size_t)(first + t0 + tb) * in.v_ld + (size_t)head * e + c]) : 0.f;
        }
        if (tid < nb) {
            const size_t at = (size_t)(first + t0 + tid) * n_heads + head;
            sg[tid] = in.log_decay != nullptr ? expf(in.log_decay[at]) : in.head_decay[head];
            if (DELTA) sb[tid] = in.beta[at];
        }
        __syncthreads();
        if (DELTA) {
            for (int tb = warp; tb < nb; tb += warps) {
                float dot = 0.f;
                for (int dd = lane; dd < ds_count * MS_R; dd += 32) {
                    const int at = tb * stride + (dd / MS_R) * (MS_R + 4) + dd % MS_R;
                    dot = fmaf(sk[at], sq[at], dot);
                }
                dot = warp_sum(dot);
                if (lane == 0) skq[tb] = dot;
            }
            __syncthreads();
        }
        for (int tb = 0; tb < nb; ++tb) {
            const float4* k4 = reinterpret_cast<const float4*>(sk + tb * stride + ds * (MS_R + 4));
            const float4* q4 = reinterpret_cast<const float4*>(sq + tb * stride + ds * (MS_R + 4));
            const float g = sg[tb], vc = owner ? sv[tb * tile_cols + local] : 0.f;
            float o;
            if (DELTA) {
                float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
#pragma unroll
                for (int r = 0; r < MS_R / 4; ++r) {
                    const float4 kk = k4[r], qq = q4[r];
                    a0 = fmaf(S[4 * r], kk.x, a0); a1 = fmaf(S[4 * r + 1], kk.y, a1);
                    b0 = fmaf(S[4 * r], qq.x, b0); b1 = fmaf(S[4 * r + 1], qq.y, b1);
                    a0 = fmaf(S[4 * r + 2], kk.z, a0); a1 = fmaf(S[4 * r + 3], kk.w, a1);
                    b0 = fmaf(S[4 * r + 2], qq.z, b0); b1 = fmaf(S[4 * r + 3], qq.w, b1);
                }
                float a = a0 + a1, b = b0 + b1;
                for (int step = 1; step < ds_count; step <<= 1) {
                    a += __shfl_xor_sync(0xffffffffu, a, step);
                    b += __shfl_xor_sync(0xffffffffu, b, step);
                }
                const float u = sb[tb] * (vc - g * a);
                o = fmaf(skq[tb], u, g * b);
#pragma unroll
                for (int r = 0; r < MS_R / 4; ++r) {
                    const float4 kk = k4[r];
                    S[4 * r] = fmaf(g, S[4 * r], kk.x * u); S[4 * r + 1] = fmaf(g, S[4 * r + 1], kk.y * u);
                    S[4 * r + 2] = fmaf(g, S[4 * r + 2], kk.z * u); S[4 * r + 3] = fmaf(g, S[4 * r + 3], kk.w * u);
                }
            } else {
                float b0 = 0.f, b1 = 0.f;
#pragma unroll
                for (int r = 0; r < MS_R / 4; ++r) {
                    const float4 kk = k4[r], qq = q4[r];
                    S[4 * r] = fmaf(g, S[4 * r], kk.x * vc); S[4 * r + 1] = fmaf(g, S[4 * r + 1], kk.y * vc);
                    S[4 * r + 2] = fmaf(g, S[4 * r + 2], kk.z * vc); S[4 * r + 3] = fmaf(g, S[4 * r + 3], kk.w * vc);
                    b0 = fmaf(S[4 * r], qq.x, b0); b1 = fmaf(S[4 * r + 1], qq.y, b1);
                    b0 = fmaf(S[4 * r + 2], qq.z, b0); b1 = fmaf(S[4 * r + 3], qq.w, b1);
                }
                o = b0 + b1;
                for (int step = 1; step < ds_count; step <<= 1) o += __shfl_xor_sync(0xffffffffu, o, step);
            }
            if (owner && ds == 0) {
                if (NORM) so[tb * tile_cols + local] = o;
                else o_raw[((size_t)(first + t0 + tb) * n_heads + head) * e + col0 + local] = o;
            }
        }
        if (NORM) {
            __syncthreads();
            head_norm_gate_rows<T, float>(so, tile_cols, nb, (size_t)(first + t0), gate, (int)gate_ld, norm_w, eps, n_heads, head,
                                          e, out, lane, warp, warps);
        }
    }
    int pitch = e;
    asm volatile("" : "+r"(pitch));        // the addresses of the loads at the top must not be kept until here
#pragma unroll
    for (int r = 0; r < MS_R; ++r)
        if (owner && ds * MS_R + r < d) slot[(size_t)r * pitch] = S[r];
}

struct StateScanShape { int ds_count, tile_cols, tiles, threads; size_t smem; };

static bool state_scan_shape(int d, int e, StateScanShape& s) {
    s.ds_count = 1;
    while (s.ds_count * MS_R < d) s.ds_count <<= 1;
    if (s.ds_count > 32) return false;
    const int most = MS_THREADS / s.ds_count;
    s.tiles = (e + most - 1) / most;
    s.tile_cols = (e + s.tiles - 1) / s.tiles;
    s.threads = (s.tile_cols * s.ds_count + 31) / 32 * 32;
    s.smem = (size_t)MS_TB * (2 * s.ds_count * (MS_R + 4) + 2 * s.tile_cols + 3) * sizeof(float);
    return s.threads <= MS_THREADS;
}

// 1: the scan leaves raw outputs for the kernel that norms rows (a head's columns take several blocks); -1: too many channels.
extern "C" int qil_state_scan_needs_scratch(int d, int e) {
    StateScanShape s;
    if (d <= 0 || e <= 0 || !state_scan_shape(d, e, s)) return -1;
    return s.tiles > 1 ? 1 : 0;
}

static int state_rows_check(const char* what, const StateRows& in, int n_heads, int d, int e, bool delta) {
    if (n_heads <= 0 || d <= 0 || e <= 0 || in.group <= 0 || n_heads % in.group)
        QIL_REFUSE("%s: heads %d (%d per q/k head) sizes %d/%d", what, n_heads, in.group, d, e);
    if ((in.log_decay == nullptr) == (in.head_decay == nullptr)) QIL_REFUSE("%s: decays per token or per head", what);
    if (delta && in.beta == nullptr) QIL_REFUSE("%s: the correction needs its step sizes", what);
    return 0;
}

// out: normed per head (norm_w float32 [e] or null) and gated (silu of `gate`'s columns, or null); with o_raw (float32 [tokens,
// heads * e]) the outputs go there as they are instead.
extern "C" int qil_state_scan(const float* q, const float* k, long long qk_ld, int group, const void* v, long long v_ld,
                              const float* log_decay, const float* head_decay, const float* beta, const void* gate,
                              long long gate_ld, const float* norm_w, float eps, float* state, const int* seg_start,
                              const int* seg_len, const int* seg_row, int n_segments, int n_heads, int d, int e, float* o_raw,
                              void* out, int act_dtype, cudaStream_t stream) {
    if (n_segments <= 0) return 0;
    const StateRows in = {q, k, qk_ld, group, v, v_ld, log_decay, head_decay, beta};
    const bool delta = beta != nullptr;
    if (state_rows_check("state_scan", in, n_heads, d, e, delta)) return -1;
    StateScanShape s;
    if (!state_scan_shape(d, e, s)) QIL_REFUSE("state_scan: %d key channels per head are more than %d", d, 32 * MS_R);
    if (n_segments > 65535) QIL_REFUSE("state_scan: %d segments", n_segments);
    if (o_raw == nullptr && s.tiles > 1) QIL_REFUSE("state_scan: %d value columns per head need the scratch buffer", e);
    if (o_raw == nullptr && out == nullptr) QIL_REFUSE("state_scan: no place for the outputs");
    const dim3 grid(n_heads * s.tiles, n_segments);
    cudaError_t err = cudaSuccess;
#define QIL_STATE_GO(DELTA, NORM)                                                                                      \
    QIL_DISPATCH_1(act_dtype, {                                                                                        \
        if (s.smem > 48 * 1024)                                                                                        \
            err = cudaFuncSetAttribute(state_scan_kernel<T, DELTA, NORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s.smem); \
        if (err == cudaSuccess)                                                                                        \
            err = qil_launch_chained(state_scan_kernel<T, DELTA, NORM>, grid, dim3(s.threads), s.smem, stream, in,     \
                                     (const T*)gate, gate_ld, norm_w, eps, state, seg_start, seg_len, seg_row,         \
                                     n_heads, d, e, s.ds_count, s.tile_cols, o_raw, (T*)out);                          \
    })
    if (delta) { if (o_raw == nullptr) QIL_STATE_GO(true, true); else QIL_STATE_GO(true, false); }
    else { if (o_raw == nullptr) QIL_STATE_GO(false, true); else QIL_STATE_GO(false, false); }
#undef QIL_STATE_GO
    if (err != cudaSuccess) { snprintf(qil_error_text, sizeof(qil_error_text), "%s", cudaGetErrorString(err)); return (int)err; }
    QIL_CHECK_LAUNCH();
}

// ------------------------------------------------------------------ chunks of long portions
extern "C" int qil_state_chunk() { return MS_CHUNK; }
extern "C" int qil_state_chunk_most_d() { return MS_MOST_D; }

// Sums of a chunk's log decays, in double: `sums` [MS_CHUNK] in shared memory; tokens past the chunk's end add nothing.  Called
// by one warp; the caller puts a barrier behind it.
__device__ __forceinline__ void chunk_log_sums(const StateRows& in, double* sums, int first, int count, int head, int n_heads,
                                               int lane) {
    if (in.head_decay != nullptr) {
        const double log_g = fmax(log((double)in.head_decay[head]), -1e30);
        for (int i = lane; i < MS_CHUNK; i += 32) sums[i] = log_g * (double)min(i + 1, count);
        return;
    }
    double before = 0.0;
#pragma unroll
    for (int part = 0; part < MS_CHUNK; part += 32) {
        const int i = part + lane;
        double x = i < count ? fmax((double)in.log_decay[(size_t)(first + i) * n_heads + head], -1e30) : 0.0;
#pragma unroll
        for (int step = 1; step < 32; step <<= 1) {
            const double other = __shfl_up_sync(0xffffffffu, x, step);
            if (lane >= step) x += other;
        }
        x += before;
        sums[i] = x;
        before = __shfl_sync(0xffffffffu, x, 31);
    }
}

__device__ __forceinline__ void ms_copy16(void* smem, const void* gmem, bool valid) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(gmem), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void ms_copy4(void* smem, const void* gmem, bool valid) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(dst), "l"(gmem), "r"(valid ? 4 : 0) : "memory");
}
__device__ __forceinline__ void ms_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void ms_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }

// MS_CHUNK rows of d floats, `ld` apart, into rows of `stride` floats; rows from `count` on and (with `pad`) columns from d up
// to dp become zero.  Rows and row stride on 16-byte boundaries take 16 bytes a copy.
__device__ __forceinline__ void ms_load_rows(float* dst, int stride, const float* src, long long ld, int count, int d, int dp,
                                             bool pad, int tid, int threads) {
    const int lane = tid & 31, warps = threads >> 5;
    if (d % 4 == 0 && ld % 4 == 0 && ((uintptr_t)src & 15) == 0) {
        for (int r = tid >> 5; r < MS_CHUNK; r += warps)         // a warp a row: no division by the row's length
            for (int c = lane * 4; c < d; c += 128) ms_copy16(dst + r * stride + c, src + (r < count ? r : 0) * ld + c, r < count);
    } else {
        for (int r = tid >> 5; r < MS_CHUNK; r += warps)
            for (int c = lane; c < d; c += 32) ms_copy4(dst + r * stride + c, src + (r < count ? r : 0) * ld + c, r < count);
    }
    if (pad && dp > d)
        for (int i = tid; i < MS_CHUNK * (dp - d); i += threads) dst[i / (dp - d) * stride + d + i % (dp - d)] = 0.f;
}

__host__ __device__ __forceinline__ int ms_padded(int d) { return (d + 15) / 16 * 16; }

// The 16 x 16 threads of a block hold X Y^T of two tiles of MS_CHUNK rows: element (ty + 16 a, tx + 16 b) in acc[a][b], b <= a
// only (what lies above the diagonal is not asked for).
__device__ __forceinline__ void ms_lower_products(const float* x, const float* y, int stride, int dp, int ty, int tx,
                                                  float (&acc)[4][4]) {
#pragma unroll
    for (int a = 0; a < 4; ++a)
#pragma unroll
        for (int b = 0; b < 4; ++b) acc[a][b] = 0.f;
    for (int c = 0; c < dp; c += 4) {
        float4 xv[4], yv[4];
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            xv[a] = *reinterpret_cast<const float4*>(x + (ty + 16 * a) * stride + c);
            yv[a] = *reinterpret_cast<const float4*>(y + (tx + 16 * a) * stride + c);
        }
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b <= a; ++b) {
                acc[a][b] = fmaf(xv[a].x, yv[b].x, acc[a][b]); acc[a][b] = fmaf(xv[a].y, yv[b].y, acc[a][b]);
                acc[a][b] = fmaf(xv[a].z, yv[b].z, acc[a][b]); acc[a][b] = fmaf(xv[a].w, yv[b].w, acc[a][b]);
            }
    }
}

#define MS_A_STRIDE 68
#define MS_DECAY_STRIDE 68       // of a (chunk, head): MS_CHUNK decays to the chunk's end, then the whole chunk's

// The decays of a chunk from every token to its end, and over all of it (one warp; sums as chunk_log_sums leaves them).
__device__ __forceinline__ void chunk_tail_decays(const double* sums, float* dst, int lane) {
    const double last = sums[MS_CHUNK - 1];
    for (int i = lane; i < MS_CHUNK; i += 32) dst[i] = expf((float)(last - sums[i]));
    if (lane == 0) dst[MS_CHUNK] = expf((float)last);
}

// (I + A)^-1 of a strictly lower A [MS_CHUNK][MS_A_STRIDE] into t (lower, zero above): the diagonal blocks of 16 by forward
// substitution, a thread per column, then blocks of 32 and of 64 from their halves, [X 0; Y Z]^-1 = [X' 0; -Z' Y X' Z'].
// tmp holds a third such tile.  All 256 threads; barriers inside and at the end.
__device__ __forceinline__ void invert_unit_lower(const float* a, float* t, float* tmp, int tid) {
    for (int i = tid; i < MS_CHUNK * MS_A_STRIDE; i += 256) t[i] = 0.f;
    __syncthreads();
    if (tid < MS_CHUNK) {
        const int base = tid / 16 * 16, col = tid % 16;
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float s = i == col ? 1.f : 0.f;
#pragma unroll
            for (int j = 0; j < i; ++j) s = fmaf(-a[(base + i) * MS_A_STRIDE + base + j], x[j], s);
            x[i] = s;
            t[(base + i) * MS_A_STRIDE + base + col] = s;
        }
    }
    __syncthreads();
#pragma unroll
    for (int half = 16; half < MS_CHUNK; half *= 2) {
        const int each = half * half;
        for (int step = 0; step < 2; ++step) {                  // tmp = Y X', then -Z' tmp
            for (int o = tid; o < MS_CHUNK / (2 * half) * each; o += 256) {
                const int base = o / each * 2 * half, i = o % each / half, j = o % half;
                const float* left = step == 0 ? a + (base + half + i) * MS_A_STRIDE + base : t + (base + half + i) * MS_A_STRIDE + base + half;
                const float* right = step == 0 ? t + base * MS_A_STRIDE + base + j : tmp + (base + half) * MS_A_STRIDE + base + j;
                float s0 = 0.f, s1 = 0.f;
                for (int c = 0; c < half; c += 2) {
                    s0 = fmaf(left[c], right[c * MS_A_STRIDE], s0);
                    s1 = fmaf(left[c + 1], right[(c + 1) * MS_A_STRIDE], s1);
                }
                if (step == 0) tmp[(base + half + i) * MS_A_STRIDE + base + j] = s0 + s1;
                else t[(base + half + i) * MS_A_STRIDE + base + j] = -(s0 + s1);
            }
            __syncthreads();
        }
    }
}

// One block per (head, chunk): U [MS_CHUNK, e] and W [MS_CHUNK, d] of the chunk (see the top), rows past its end zero, and the
// decays to the chunk's end.
template <typename T>
__global__ void __launch_bounds__(256, 2)
delta_solve_kernel(StateRows in, const int* __restrict__ chunk_start, const int* __restrict__ chunk_len, int n_heads, int d, int e,
                   float* __restrict__ u_out, float* __restrict__ w_out, float* __restrict__ decays) {
    extern __shared__ __align__(16) float smem[];
    __shared__ double sums[MS_CHUNK];
    __shared__ float beta[MS_CHUNK], beta_decay[MS_CHUNK];
    const int dp = ms_padded(d), stride = dp + 4;
    float* sk = smem;                           // [MS_CHUNK][stride]
    float* sa = sk + MS_CHUNK * stride;         // [MS_CHUNK][MS_A_STRIDE]: A
    float* st = sa + MS_CHUNK * MS_A_STRIDE;    // the same: its inverse
    float* sv = st + MS_CHUNK * MS_A_STRIDE;    // the same: scratch, then 64 columns of values
    const int head = blockIdx.x, chunk = blockIdx.y, tid = threadIdx.x;
    const int first = chunk_start[chunk], count = chunk_len[chunk];
    const size_t block = (size_t)chunk * n_heads + head;
    qil_wait_for_producer();
    qil_release_consumer();
    ms_load_rows(sk, stride, in.k + (size_t)first * in.qk_ld + (size_t)(head / in.group) * d, in.qk_ld, count, d, dp, true, tid, 256);
    ms_commit();
    if (tid < 32) chunk_log_sums(in, sums, first, count, head, n_heads, tid);
    ms_wait<0>();
    __syncthreads();
    if (tid < MS_CHUNK) {
        const float b = tid < count ? in.beta[(size_t)(first + tid) * n_heads + head] : 0.f;
        beta[tid] = b;
        beta_decay[tid] = b * expf((float)sums[tid]);
    } else if (tid >= 224) {
        chunk_tail_decays(sums, decays + block * MS_DECAY_STRIDE, tid & 31);
    }
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;
    {
        float acc[4][4];
        ms_lower_products(sk, sk, stride, dp, ty, tx, acc);
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b) {
                const int i = ty + 16 * a, j = tx + 16 * b;
                sa[i * MS_A_STRIDE + j] = (b <= a && j < i) ? beta[i] * expf((float)(sums[i] - sums[j])) * acc[a][b] : 0.f;
            }
    }
    __syncthreads();
    invert_unit_lower(sa, st, sv, tid);
    for (int r = tid >> 5; r < MS_CHUNK; r += 8)                  // the keys' right side
        for (int c = tid & 31; c < dp; c += 32) sk[r * stride + c] *= beta_decay[r];
    const T* v = reinterpret_cast<const T*>(in.v);
    for (int tile = 0; tile < (e + 63) / 64 + (d + 63) / 64; ++tile) {
        const bool is_value = tile < (e + 63) / 64;
        const int col0 = (is_value ? tile : tile - (e + 63) / 64) * 64, width = is_value ? e : d;
        if (is_value) {
            __syncthreads();            // the tile before has been read
#pragma unroll 8
            for (int i = tid; i < MS_CHUNK * 64; i += 256) {
                const int r = i / 64, c = col0 + i % 64;
                sv[r * MS_A_STRIDE + i % 64] = (r < count && c < e)
                    ? beta[r] * to_f32<T>(v[(size_t)(first + r) * in.v_ld + (size_t)head * e + c]) : 0.f;
            }
        }
        __syncthreads();
        const float* right = is_value ? sv + 4 * tx : sk + col0 + 4 * tx;
        const int right_stride = is_value ? MS_A_STRIDE : stride;
        const bool real = is_value || col0 + 4 * tx < dp;
        float acc[4][4];
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b) acc[a][b] = 0.f;
#pragma unroll
        for (int jb = 0; jb < 4; ++jb)         // rows of block a read columns of blocks up to a
#pragma unroll 2
            for (int c = 16 * jb; c < 16 * jb + 16 && real; c += 4) {
                float4 xv[4];
#pragma unroll
                for (int a = jb; a < 4; ++a) xv[a] = *reinterpret_cast<const float4*>(st + (ty + 16 * a) * MS_A_STRIDE + c);
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    const float4 b = *reinterpret_cast<const float4*>(right + (c + r) * right_stride);
#pragma unroll
                    for (int a = jb; a < 4; ++a) {
                        const float x = r == 0 ? xv[a].x : r == 1 ? xv[a].y : r == 2 ? xv[a].z : xv[a].w;
                        acc[a][0] = fmaf(x, b.x, acc[a][0]); acc[a][1] = fmaf(x, b.y, acc[a][1]);
                        acc[a][2] = fmaf(x, b.z, acc[a][2]); acc[a][3] = fmaf(x, b.w, acc[a][3]);
                    }
                }
            }
        float* dst = (is_value ? u_out : w_out) + block * MS_CHUNK * width + col0 + 4 * tx;
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            float* at = dst + (size_t)(ty + 16 * a) * width;
            if (width % 4 == 0 && col0 + 4 * tx + 3 < width) {
                *reinterpret_cast<float4*>(at) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
            } else {
#pragma unroll
                for (int b = 0; b < 4; ++b) if (col0 + 4 * tx + b < width) at[b] = acc[a][b];
            }
        }
    }
}

// ------------------------------------------------------------------ the chunks of a portion in order
// MS_CHUNK rows of d floats, `ld` apart, into rows of DP + 16 floats by 256 threads; rows from `count` on become zero, columns from
// d on stay as they are.
template <int DP>
__device__ __forceinline__ void ms_load_tile(float* dst, const float* src, long long ld, int count, int d, int tid) {
    if (d % 4 != 0 || ld % 4 != 0 || ((uintptr_t)src & 15) != 0) {
        ms_load_rows(dst, DP + 16, src, ld, count, d, DP, false, tid, 256);
        return;
    }
    constexpr int PIECES = DP / 4, ROWS = 256 / PIECES;
    const int r0 = tid / PIECES, c = tid % PIECES * 4;
    if (c >= d) return;
    const float* from = src + r0 * ld + c;
    const long long step = ROWS * ld;
#pragma unroll
    for (int n = 0; n < MS_CHUNK / ROWS; ++n) {
        const bool real = r0 + n * ROWS < count;
        ms_copy16(dst + (r0 + n * ROWS) * (DP + 16) + c, real ? from : src, real);
        from += step;
    }
}

// Sums of 16 values over LANES neighbouring lanes; lane l of them keeps values l * 16 / LANES and following, at the front.
template <int LANES>
__device__ __forceinline__ void scatter_sums(float (&v)[16], int lane) {
    int n = 16;
#pragma unroll
    for (int step = LANES / 2; step > 0; step >>= 1) {
        n >>= 1;
        const bool upper = (lane & step) != 0;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (i >= n) break;
            const float other = __shfl_xor_sync(0xffffffffu, upper ? v[i] : v[i + n], step);
            v[i] = (upper ? v[i + n] : v[i]) + other;
        }
    }
}

// One block per (head, COLS value columns, long portion).  carry: int32 [portions, 3] = (state slot, first chunk, chunks).
// chunk_state [chunks, heads, d, e] receives the state that comes into every chunk, y [chunks, heads, MS_CHUNK, e] the
// corrected values in place of u; the state after the last chunk goes to the request's slot.  The state's columns live in
// registers, with a copy in shared memory for the first product.  DP: key channels that the tiles hold, at least d; the rest
// stays zero.
template <int COLS, int DP>
__global__ void __launch_bounds__(256, 1)
delta_walk_kernel(StateRows in, const int* __restrict__ chunk_start, const int* __restrict__ chunk_len, const int* __restrict__ carry,
                  int n_heads, int d, int e, float* __restrict__ y, const float* __restrict__ w_in, const float* __restrict__ decays,
                  float* __restrict__ chunk_state, float* __restrict__ slots, int stages) {
    constexpr int CG = COLS / 4;           // groups of four columns
    constexpr int KS = 16 / CG;            // lanes that share 4 x 4 elements of the first product, each over a part of the channels
    constexpr int TS = 8 / CG;             // the same for the second product, over the tokens
    constexpr int KEEP = 16 / KS, HOLD = 16 / TS;
    constexpr int ITEMS = (DP + 127) / 128;                            // of 128 channels that a thread serves
    constexpr int STRIDE = DP + 16, STATE_STRIDE = DP + 4, TILE = MS_CHUNK * STRIDE;      // 16 banks from row to row
    extern __shared__ __align__(16) float smem[];
    float* sk = smem;                                  // [stages][MS_CHUNK][STRIDE]
    float* sw = sk + stages * TILE;                    // the same
    float* ss = sw + stages * TILE;                    // [COLS][STATE_STRIDE]
    float* sy = ss + COLS * STATE_STRIDE;              // [MS_CHUNK][COLS]: y times its decay to the chunk's end
    float* sd = sy + MS_CHUNK * COLS;                  // [stages][MS_DECAY_STRIDE]
    const int tiles = (e + COLS - 1) / COLS;
    const int head = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * COLS, tid = threadIdx.x;
    const int row = carry[3 * blockIdx.y], chunk0 = carry[3 * blockIdx.y + 1], chunks = carry[3 * blockIdx.y + 2];
    const size_t qk_at = (size_t)(head / in.group) * d;
    const int total = stages * (2 * TILE + MS_DECAY_STRIDE) + COLS * (STATE_STRIDE + MS_CHUNK);
    for (int i = tid; i < total; i += 256) smem[i] = 0.f;      // the padding stays zero
    const int part = tid % KS, cg = tid / KS % CG, rg = tid / KS / CG;                  // first product: rows rg + 16 a
    const int my_row = rg + 16 * (part * KEEP / 4), my_col = 4 * cg + part * KEEP % 4;  // of the sums this thread keeps
    const int ts = tid % TS, gc = tid / TS % CG, d_first = tid / TS / CG * 4;           // second product: channels d_first + 128 it
    const int hold_d = ts * HOLD / 4;                                                   // of the sums this thread keeps: HOLD / 4 channels
    const bool aligned = e % 4 == 0 && col0 + COLS <= e;
    qil_wait_for_producer();
    qil_release_consumer();
    __syncthreads();
    float S[ITEMS][HOLD];
    float* slot = slots + ((size_t)row * n_heads + head) * d * e + col0 + 4 * gc;
#pragma unroll
    for (int it = 0; it < ITEMS; ++it)
#pragma unroll
        for (int i = 0; i < HOLD; ++i) {
            const int dd = d_first + 128 * it + hold_d + i / 4;
            S[it][i] = (dd < d && col0 + 4 * gc + i % 4 < e) ? slot[(size_t)dd * e + i % 4] : 0.f;
            if (dd < DP) ss[(4 * gc + i % 4) * STATE_STRIDE + dd] = S[it][i];
        }
    auto fetch = [&](int chunk, int stage) {
        const int first = chunk_start[chunk], count = chunk_len[chunk];
        const size_t block = (size_t)chunk * n_heads + head;
        ms_load_tile<DP>(sk + stage * TILE, in.k + (size_t)first * in.qk_ld + qk_at, in.qk_ld, count, d, tid);
        ms_load_tile<DP>(sw + stage * TILE, w_in + block * MS_CHUNK * d, d, MS_CHUNK, d, tid);
        if (tid < MS_DECAY_STRIDE / 4) ms_copy16(sd + stage * MS_DECAY_STRIDE + 4 * tid, decays + block * MS_DECAY_STRIDE + 4 * tid, true);
        ms_commit();
    };
    auto at_y = [&](int chunk) { return y + (((size_t)chunk * n_heads + head) * MS_CHUNK + my_row) * e + col0 + my_col; };
    auto read_u = [&](int chunk, float (&u)[KEEP]) {
        const float* p = at_y(chunk);
        if (aligned && KEEP == 4) {
            const float4 q = *reinterpret_cast<const float4*>(p);
            u[0] = q.x; u[1 % KEEP] = q.y; u[2 % KEEP] = q.z; u[3 % KEEP] = q.w;
        } else if (aligned && KEEP == 2) {
            const float2 q = *reinterpret_cast<const float2*>(p);
            u[0] = q.x; u[1 % KEEP] = q.y;
        } else {
#pragma unroll
            for (int i = 0; i < KEEP; ++i) u[i] = col0 + my_col + i < e ? p[i] : 0.f;
        }
    };
    float u[KEEP];
    read_u(chunk0, u);
    if (stages == 2) fetch(chunk0, 0);
    for (int n = 0; n < chunks; ++n) {
        const int chunk = chunk0 + n, stage = stages == 2 ? (n & 1) : 0;
        if (stages == 1) fetch(chunk, 0);
        ms_wait<0>();
        __syncthreads();                   // this chunk's tiles are here, everyone has left the chunk before
        if (stages == 2 && n + 1 < chunks) fetch(chunk + 1, stage ^ 1);
        const float* tk = sk + stage * TILE;
        const float* tw = sw + stage * TILE;
        const float* tail = sd + stage * MS_DECAY_STRIDE;
        float* into = chunk_state + ((size_t)chunk * n_heads + head) * d * e + col0 + 4 * gc;
#pragma unroll
        for (int it = 0; it < ITEMS; ++it)
#pragma unroll
            for (int i = 0; i < HOLD; i += 4) {
                const int dd = d_first + 128 * it + hold_d + i / 4;
                if (dd >= d) continue;
                if (aligned) {
                    *reinterpret_cast<float4*>(into + (size_t)dd * e) = make_float4(S[it][i], S[it][i + 1], S[it][i + 2], S[it][i + 3]);
                } else {
#pragma unroll
                    for (int b = 0; b < 4; ++b) if (col0 + 4 * gc + b < e) into[(size_t)dd * e + b] = S[it][i + b];
                }
            }
        {
            float acc[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) acc[i] = 0.f;
            const float* w_at = tw + rg * STRIDE + part * 4;
            const float* s_at = ss + 4 * cg * STATE_STRIDE + part * 4;
#pragma unroll 4
            for (int c = 0; c < DP; c += 4 * KS) {
                float4 wv[4], sv[4];
#pragma unroll
                for (int a = 0; a < 4; ++a) {
                    wv[a] = *reinterpret_cast<const float4*>(w_at + 16 * a * STRIDE + c);
                    sv[a] = *reinterpret_cast<const float4*>(s_at + a * STATE_STRIDE + c);
                }
#pragma unroll
                for (int a = 0; a < 4; ++a)
#pragma unroll
                    for (int b = 0; b < 4; ++b) {
                        acc[4 * a + b] = fmaf(wv[a].x, sv[b].x, acc[4 * a + b]); acc[4 * a + b] = fmaf(wv[a].y, sv[b].y, acc[4 * a + b]);
                        acc[4 * a + b] = fmaf(wv[a].z, sv[b].z, acc[4 * a + b]); acc[4 * a + b] = fmaf(wv[a].w, sv[b].w, acc[4 * a + b]);
                    }
            }
            scatter_sums<KS>(acc, part);
            const float decay = tail[my_row];
            float* p = at_y(chunk);
#pragma unroll
            for (int i = 0; i < KEEP; ++i) {
                u[i] -= acc[i];
                sy[my_row * COLS + my_col + i] = u[i] * decay;
            }
            if (aligned && KEEP == 4) {
                *reinterpret_cast<float4*>(p) = make_float4(u[0], u[1 % KEEP], u[2 % KEEP], u[3 % KEEP]);
            } else if (aligned && KEEP == 2) {
                *reinterpret_cast<float2*>(p) = make_float2(u[0], u[1 % KEEP]);
            } else {
#pragma unroll
                for (int i = 0; i < KEEP; ++i) if (col0 + my_col + i < e) p[i] = u[i];
            }
            if (n + 1 < chunks) read_u(chunk + 1, u);
        }
        const float whole = tail[MS_CHUNK];
        __syncthreads();                   // y is here, everyone has read the state's columns
#pragma unroll
        for (int it = 0; it < ITEMS; ++it) {
            const int d4 = d_first + 128 * it;
            if (d4 >= DP) break;           // whole warps leave together
            float acc[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) acc[i] = 0.f;
            const float* k_at = tk + ts * STRIDE + d4;
            const float* y_at = sy + ts * COLS + 4 * gc;
#pragma unroll 8
            for (int t = 0; t < MS_CHUNK; t += TS) {
                const float4 kv = *reinterpret_cast<const float4*>(k_at + t * STRIDE);
                const float4 yv = *reinterpret_cast<const float4*>(y_at + t * COLS);
                const float ka[4] = {kv.x, kv.y, kv.z, kv.w}, ya[4] = {yv.x, yv.y, yv.z, yv.w};
#pragma unroll
                for (int a = 0; a < 4; ++a)
#pragma unroll
                    for (int b = 0; b < 4; ++b) acc[4 * a + b] = fmaf(ka[a], ya[b], acc[4 * a + b]);
            }
            scatter_sums<TS>(acc, ts);
#pragma unroll
            for (int i = 0; i < HOLD; ++i) {
                S[it][i] = fmaf(whole, S[it][i], acc[i]);
                ss[(4 * gc + i % 4) * STATE_STRIDE + d4 + hold_d + i / 4] = S[it][i];
            }
        }
        if (stages == 1) __syncthreads();  // the tiles are overwritten next
    }
#pragma unroll
    for (int it = 0; it < ITEMS; ++it)
#pragma unroll
        for (int i = 0; i < HOLD; ++i) {
            const int dd = d_first + 128 * it + hold_d + i / 4;
            if (dd < d && col0 + 4 * gc + i % 4 < e) slot[(size_t)dd * e + i % 4] = S[it][i];
        }
}

// Without the correction a chunk's own state needs no state: sum_j e^(L_C - L_j) k_j v_j^T for all chunks at once (chunk_state
// [chunks, heads, d, e]) and the chunk's decay for every channel (decay_product [chunks, heads, d]); gla_carry walks them.
// One block per (head, chunk, 64 value columns).
template <typename T>
__global__ void __launch_bounds__(256)
state_own_kernel(StateRows in, const int* __restrict__ chunk_start, const int* __restrict__ chunk_len, int n_heads, int d, int e,
                 float* __restrict__ chunk_state, float* __restrict__ decay_product) {
    extern __shared__ __align__(16) float smem[];
    __shared__ double sums[MS_CHUNK];
    __shared__ float tail[MS_DECAY_STRIDE];
    const int dp = ms_padded(d), stride = dp + 4;
    float* sk = smem;                           // [MS_CHUNK][stride]
    float* sv = sk + MS_CHUNK * stride;         // [MS_CHUNK][MS_A_STRIDE]
    const int head = blockIdx.x, chunk = blockIdx.y, col0 = blockIdx.z * 64, tid = threadIdx.x;
    const int first = chunk_start[chunk], count = chunk_len[chunk];
    const size_t block = (size_t)chunk * n_heads + head;
    const T* v = reinterpret_cast<const T*>(in.v);
    qil_wait_for_producer();
    qil_release_consumer();
    ms_load_rows(sk, stride, in.k + (size_t)first * in.qk_ld + (size_t)(head / in.group) * d, in.qk_ld, count, d, dp, true, tid, 256);
    ms_commit();
    if (tid < 32) {
        chunk_log_sums(in, sums, first, count, head, n_heads, tid);
        __syncwarp();
        chunk_tail_decays(sums, tail, tid);
    }
    __syncthreads();
#pragma unroll 8
    for (int i = tid; i < MS_CHUNK * 64; i += 256) {
        const int r = i / 64, c = col0 + i % 64;
        sv[r * MS_A_STRIDE + i % 64] = (r < count && c < e) ? tail[r] * to_f32<T>(v[(size_t)(first + r) * in.v_ld + (size_t)head * e + c]) : 0.f;
    }
    if (blockIdx.z == 0)
        for (int i = tid; i < d; i += 256) decay_product[block * d + i] = tail[MS_CHUNK];
    ms_wait<0>();
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;
    for (int d4 = 4 * ty; d4 < dp; d4 += 64) {
        float acc[4][4];
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b) acc[a][b] = 0.f;
#pragma unroll 8
        for (int t = 0; t < MS_CHUNK; ++t) {
            const float4 kv = *reinterpret_cast<const float4*>(sk + t * stride + d4);
            const float4 yv = *reinterpret_cast<const float4*>(sv + t * MS_A_STRIDE + 4 * tx);
            const float ka[4] = {kv.x, kv.y, kv.z, kv.w}, ya[4] = {yv.x, yv.y, yv.z, yv.w};
#pragma unroll
            for (int a = 0; a < 4; ++a)
#pragma unroll
                for (int b = 0; b < 4; ++b) acc[a][b] = fmaf(ka[a], ya[b], acc[a][b]);
        }
        const int c = col0 + 4 * tx;
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            if (d4 + a >= d) break;
            float* dst = chunk_state + (block * d + d4 + a) * e + c;
            if (e % 4 == 0 && c + 3 < e) {
                *reinterpret_cast<float4*>(dst) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
            } else {
#pragma unroll
                for (int b = 0; b < 4; ++b) if (c + b < e) dst[b] = acc[a][b];
            }
        }
    }
}

// ------------------------------------------------------------------ the outputs of all chunks
// One block per (head, chunk): raw outputs float32 [tokens, heads * e].
#define MS_OUT_COLS 64
template <typename T, bool DELTA>
__global__ void __launch_bounds__(256)
state_outputs_kernel(StateRows in, const int* __restrict__ chunk_start, const int* __restrict__ chunk_len, int n_heads, int d, int e,
                     const float* __restrict__ y, const float* __restrict__ chunk_state, float* __restrict__ o_raw) {
    extern __shared__ __align__(16) float smem[];
    __shared__ double sums[MS_CHUNK];
    const int dp = ms_padded(d), stride = dp + 4;
    float* sq = smem;                                  // [MS_CHUNK][stride]
    float* sm = sq + MS_CHUNK * stride;                // [MS_CHUNK][MS_A_STRIDE]
    float* sk = sm + MS_CHUNK * MS_A_STRIDE;           // [MS_CHUNK][stride], then:
    float* ss = sk;                                    // [dp][MS_OUT_COLS]
    float* sy = ss + dp * MS_OUT_COLS;                 // [MS_CHUNK][MS_OUT_COLS]
    const int head = blockIdx.x, chunk = blockIdx.y, tid = threadIdx.x;
    const int first = chunk_start[chunk], count = chunk_len[chunk];
    const size_t qk_at = (size_t)(head / in.group) * d;
    qil_wait_for_producer();
    qil_release_consumer();
    ms_load_rows(sq, stride, in.q + (size_t)first * in.qk_ld + qk_at, in.qk_ld, count, d, dp, true, tid, 256);
    ms_load_rows(sk, stride, in.k + (size_t)first * in.qk_ld + qk_at, in.qk_ld, count, d, dp, true, tid, 256);
    ms_commit();
    if (tid < 32) chunk_log_sums(in, sums, first, count, head, n_heads, tid);
    ms_wait<0>();
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;
    {
        float acc[4][4];
        ms_lower_products(sq, sk, stride, dp, ty, tx, acc);
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b) {
                const int i = ty + 16 * a, j = tx + 16 * b;
                sm[i * MS_A_STRIDE + j] = (b <= a && j <= i) ? expf((float)(sums[i] - sums[j])) * acc[a][b] : 0.f;
            }
    }
    float decay[4];
#pragma unroll
    for (int a = 0; a < 4; ++a) decay[a] = expf((float)sums[ty + 16 * a]);
    const T* v = reinterpret_cast<const T*>(in.v);
    const size_t block = (size_t)chunk * n_heads + head;
    for (int col0 = 0; col0 < e; col0 += MS_OUT_COLS) {
        __syncthreads();                    // the keys, or the tile before, have been read
        const float* from = chunk_state + block * d * e + col0;
        const bool wide = e % 4 == 0 && col0 + MS_OUT_COLS <= e;
        if (wide) {
            for (int i = tid; i < d * (MS_OUT_COLS / 4); i += 256)
                ms_copy16(ss + i * 4, from + (size_t)(i / (MS_OUT_COLS / 4)) * e + i % (MS_OUT_COLS / 4) * 4, true);
        } else {
            for (int i = tid; i < d * MS_OUT_COLS; i += 256) {
                const int dd = i / MS_OUT_COLS, c = i % MS_OUT_COLS;
                const bool real = col0 + c < e;
                ms_copy4(ss + i, real ? from + (size_t)dd * e + c : from, real);
            }
        }
        for (int i = tid; i < (dp - d) * MS_OUT_COLS; i += 256) ss[d * MS_OUT_COLS + i] = 0.f;
        if (DELTA) {
            const float* rows = y + block * MS_CHUNK * e + col0;
            if (wide) {
                for (int i = tid; i < MS_CHUNK * (MS_OUT_COLS / 4); i += 256)
                    ms_copy16(sy + i * 4, rows + (size_t)(i / (MS_OUT_COLS / 4)) * e + i % (MS_OUT_COLS / 4) * 4, true);
            } else {
                for (int i = tid; i < MS_CHUNK * MS_OUT_COLS; i += 256) {
                    const int t = i / MS_OUT_COLS, c = i % MS_OUT_COLS;
                    const bool real = col0 + c < e;
                    ms_copy4(sy + i, real ? rows + (size_t)t * e + c : rows, real);
                }
            }
        } else {
#pragma unroll 8
            for (int i = tid; i < MS_CHUNK * MS_OUT_COLS; i += 256) {
                const int t = i / MS_OUT_COLS, c = col0 + i % MS_OUT_COLS;
                sy[i] = (t < count && c < e) ? to_f32<T>(v[(size_t)(first + t) * in.v_ld + (size_t)head * e + c]) : 0.f;
            }
        }
        ms_commit();
        ms_wait<0>();
        __syncthreads();
        float acc[4][4];
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b) acc[a][b] = 0.f;
        auto gather = [&](const float* left, int left_stride, const float* right, int depth) {
#pragma unroll 2
            for (int c = 0; c < depth; c += 4) {
                float4 xv[4];
#pragma unroll
                for (int a = 0; a < 4; ++a) xv[a] = *reinterpret_cast<const float4*>(left + (ty + 16 * a) * left_stride + c);
#pragma unroll
                for (int r = 0; r < 4; ++r) {
                    const float4 b = *reinterpret_cast<const float4*>(right + (c + r) * MS_OUT_COLS + 4 * tx);
#pragma unroll
                    for (int a = 0; a < 4; ++a) {
                        const float x = r == 0 ? xv[a].x : r == 1 ? xv[a].y : r == 2 ? xv[a].z : xv[a].w;
                        acc[a][0] = fmaf(x, b.x, acc[a][0]); acc[a][1] = fmaf(x, b.y, acc[a][1]);
                        acc[a][2] = fmaf(x, b.z, acc[a][2]); acc[a][3] = fmaf(x, b.w, acc[a][3]);
                    }
                }
            }
        };
        gather(sq, stride, ss, dp);
#pragma unroll
        for (int a = 0; a < 4; ++a)
#pragma unroll
            for (int b = 0; b < 4; ++b) acc[a][b] *= decay[a];
        gather(sm, MS_A_STRIDE, sy, (count + 3) / 4 * 4);
#pragma unroll
        for (int a = 0; a < 4; ++a) {
            const int i = ty + 16 * a, c = col0 + 4 * tx;
            if (i >= count) continue;
            float* dst = o_raw + ((size_t)(first + i) * n_heads + head) * e + c;
            if (wide) {
                *reinterpret_cast<float4*>(dst) = make_float4(acc[a][0], acc[a][1], acc[a][2], acc[a][3]);
            } else {
#pragma unroll
                for (int b = 0; b < 4; ++b) if (c + b < e) dst[b] = acc[a][b];
            }
        }
    }
}

template <typename Kernel>
static cudaError_t ms_reserve(Kernel kernel, size_t smem) {
    // the default limit of 48 KB counts the kernels' static arrays too
    return smem > 40 * 1024 ? cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : cudaSuccess;
}

extern "C" int qil_gla_carry(float* chunk_state, const float* decay_product, float* slots, const int* carry, int n_carries,
                             int n_heads, int d, int e, cudaStream_t stream);

static int delta_walk_dp(int d) { return d <= 64 ? 64 : d <= 128 ? 128 : MS_MOST_D; }
static size_t delta_walk_smem(int d, int cols, int stages) {
    const int dp = delta_walk_dp(d);
    return (size_t)(stages * (2 * MS_CHUNK * (dp + 16) + MS_DECAY_STRIDE) + cols * (dp + 4 + MS_CHUNK)) * sizeof(float);
}

// Floats of scratch per (chunk, head) that qil_state_chunks wants beside the chunks' states: with the correction U, W and the
// decays, without it a decay per channel.
extern "C" int qil_state_chunk_scratch(int d, int e, int delta) {
    return delta ? MS_CHUNK * (d + e) + MS_DECAY_STRIDE : d;
}

// The chunked form over a step's long portions.  scratch: float32 [chunks * heads * qil_state_chunk_scratch]; chunk_state float32
// [chunks, heads, d, e]: scratch too.  o_raw float32 [tokens, heads * e]: the outputs of the chunks' tokens, as they are.
extern "C" int qil_state_chunks(const float* q, const float* k, long long qk_ld, int group, const void* v, long long v_ld,
                                const float* log_decay, const float* head_decay, const float* beta, const int* chunk_start,
                                const int* chunk_len, int n_chunks, const int* carry, int n_carries, int n_heads, int d, int e,
                                float* scratch, float* chunk_state, float* slots, float* o_raw, int act_dtype, cudaStream_t stream) {
    if (n_chunks <= 0) return 0;
    const StateRows in = {q, k, qk_ld, group, v, v_ld, log_decay, head_decay, beta};
    const bool delta = beta != nullptr;
    if (state_rows_check("state_chunks", in, n_heads, d, e, delta)) return -1;
    if (d > MS_MOST_D) QIL_REFUSE("state_chunks: %d key channels per head are more than %d", d, MS_MOST_D);
    if (n_chunks > 65535 || n_carries <= 0 || n_carries > 65535) QIL_REFUSE("state_chunks: %d chunks of %d portions", n_chunks, n_carries);
    if (scratch == nullptr || ((uintptr_t)scratch & 15) != 0 || ((uintptr_t)chunk_state & 15) != 0)
        QIL_REFUSE("state_chunks: scratch on 16-byte boundaries");
    const int dp = ms_padded(d);
    const size_t row_tile = (size_t)MS_CHUNK * (dp + 4) * sizeof(float), a_tile = (size_t)MS_CHUNK * MS_A_STRIDE * sizeof(float);
    const size_t after_keys = (size_t)(dp + MS_CHUNK) * MS_OUT_COLS * sizeof(float);
    const size_t out_smem = row_tile + a_tile + (row_tile > after_keys ? row_tile : after_keys);
    const size_t pairs = (size_t)n_chunks * n_heads;
    // the decays first: their stride is a multiple of four, so that all three parts can start on 16-byte boundaries
    float* decays = scratch;
    float* y = decays + (delta ? pairs * MS_DECAY_STRIDE : 0);
    float* w = y + (delta ? pairs * MS_CHUNK * e : 0);
    // few columns a block where that still leaves every block a multiprocessor of its own
    const int cols = (long long)n_heads * ((e + 7) / 8) * n_carries <= 148 ? 8 : 16;
    const int tiles = (e + cols - 1) / cols;
    const int stages = delta_walk_smem(d, cols, 2) <= 200 * 1024 ? 2 : 1;
    const size_t walk_smem = delta_walk_smem(d, cols, stages);
    cudaError_t err = cudaSuccess;
#define QIL_MS(...) do { if (err == cudaSuccess) err = (__VA_ARGS__); } while (0)
#define QIL_MS_WALK(COLS, DP)                                                                                           \
    do {                                                                                                                \
        QIL_MS(ms_reserve(delta_walk_kernel<COLS, DP>, walk_smem));                                                     \
        QIL_MS(qil_launch_chained(delta_walk_kernel<COLS, DP>, dim3(n_heads * tiles, n_carries), dim3(256), walk_smem, stream,  \
                                  in, chunk_start, chunk_len, carry, n_heads, d, e, y, (const float*)w, (const float*)decays,   \
                                  chunk_state, slots, stages));                                                         \
    } while (0)
#define QIL_MS_COLS(DP) do { if (cols == 8) QIL_MS_WALK(8, DP); else QIL_MS_WALK(16, DP); } while (0)
#define QIL_MS_OUTPUTS(DELTA)                                                                                           \
    do {                                                                                                                \
        QIL_MS(ms_reserve(state_outputs_kernel<T, DELTA>, out_smem));                                                   \
        QIL_MS(qil_launch_chained(state_outputs_kernel<T, DELTA>, dim3(n_heads, n_chunks), dim3(256), out_smem, stream, in, \
                                  chunk_start, chunk_len, n_heads, d, e, (const float*)y, (const float*)chunk_state, o_raw)); \
    } while (0)
    QIL_DISPATCH_1(act_dtype, {
        if (delta) {
            QIL_MS(ms_reserve(delta_solve_kernel<T>, row_tile + 3 * a_tile));
            QIL_MS(qil_launch_chained(delta_solve_kernel<T>, dim3(n_heads, n_chunks), dim3(256), row_tile + 3 * a_tile, stream, in,
                                      chunk_start, chunk_len, n_heads, d, e, y, w, decays));
            if (delta_walk_dp(d) == 64) QIL_MS_COLS(64);
            else if (delta_walk_dp(d) == 128) QIL_MS_COLS(128);
            else QIL_MS_COLS(MS_MOST_D);
            QIL_MS_OUTPUTS(true);
        } else {
            QIL_MS(ms_reserve(state_own_kernel<T>, row_tile + a_tile));
            QIL_MS(qil_launch_chained(state_own_kernel<T>, dim3(n_heads, n_chunks, (e + 63) / 64), dim3(256), row_tile + a_tile, stream,
                                      in, chunk_start, chunk_len, n_heads, d, e, chunk_state, decays));
            if (err == cudaSuccess) {
                const int code = qil_gla_carry(chunk_state, decays, slots, carry, n_carries, n_heads, d, e, stream);
                if (code != 0) return code;
            }
            QIL_MS_OUTPUTS(false);
        }
    });
#undef QIL_MS_OUTPUTS
#undef QIL_MS_COLS
#undef QIL_MS_WALK
#undef QIL_MS
    if (err != cudaSuccess) { snprintf(qil_error_text, sizeof(qil_error_text), "%s", cudaGetErrorString(err)); return (int)err; }
    QIL_CHECK_LAUNCH();
}

// ------------------------------------------------------------------ what the delta rule reads
// The tail of a gated delta rule's projection.  Per token: q and k [kv_heads * d], v [heads * e] are the first columns of its
// row, each channel through a short causal convolution over time (taps_w float32 [taps][channels], as in short_conv.cu; earlier
// rows of other steps from the request's slot float32 [taps - 1][channels]) and silu; q and k then become unit vectors per
// head, x / sqrt(sum x^2 + 1e-6), q times q_scale: float32 rows qk [tokens, 2 * kv_heads * d] (q, then k); v goes to v_out in
// the activations' type.  beta = sigmoid(b), log_decay = -exp(A_log) softplus(a + dt_bias): float32 [tokens, heads].  A
// request's only token of a step moves its slot on by one row here; slots of longer segments move in short_conv_state.
#define MS_PREPARE_KEPT 8        // values of a head that a lane keeps in registers
template <int V> struct MsVec { float x[V]; };
template <typename T, int V> __device__ __forceinline__ MsVec<V> ms_read(const T* p);
template <> __device__ __forceinline__ MsVec<1> ms_read<float, 1>(const float* p) { return {{p[0]}}; }
template <> __device__ __forceinline__ MsVec<1> ms_read<bf16, 1>(const bf16* p) { return {{to_f32<bf16>(p[0])}}; }
template <> __device__ __forceinline__ MsVec<4> ms_read<float, 4>(const float* p) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    return {{v.x, v.y, v.z, v.w}};
}
template <> __device__ __forceinline__ MsVec<4> ms_read<bf16, 4>(const bf16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return {{lo.x, lo.y, hi.x, hi.y}};
}
__device__ __forceinline__ void ms_write(float* p, const MsVec<1>& v) { p[0] = v.x[0]; }
__device__ __forceinline__ void ms_write(bf16* p, const MsVec<1>& v) { p[0] = from_f32<bf16>(v.x[0]); }
__device__ __forceinline__ void ms_write(float* p, const MsVec<4>& v) {
    *reinterpret_cast<float4*>(p) = make_float4(v.x[0], v.x[1], v.x[2], v.x[3]);
}
__device__ __forceinline__ void ms_write(bf16* p, const MsVec<4>& v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x[0], v.x[1]), hi = __floats2bfloat162_rn(v.x[2], v.x[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const unsigned*>(&lo);
    raw.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
}

struct DeltaInputs {
    long long ld;
    int b_col, a_col;
    const float* taps_w;
    int taps;
    float* state;
    const float* a_log;
    const float* dt_bias;
    float q_scale;
    const int* positions;
    const int* token_row;
    int n_tokens, heads, kv_heads, d, e;
    float* qk;
    float* beta;
    float* log_decay;
};

template <typename T>
__device__ __forceinline__ void delta_gates(const DeltaInputs& in, const T* row, int token, int lane) {
    for (int h = lane; h < in.heads; h += 32) {
        const float b = to_f32<T>(row[in.b_col + h]), a = to_f32<T>(row[in.a_col + h]) + in.dt_bias[h];
        in.beta[(size_t)token * in.heads + h] = 1.f / (1.f + expf(-b));
        const float softplus = fmaxf(a, 0.f) + log1pf(expf(-fabsf(a)));
        in.log_decay[(size_t)token * in.heads + h] = -expf(in.a_log[h]) * softplus;
    }
}

__device__ __forceinline__ float ms_silu(float y) { return y / (1.f + expf(-y)); }

// One token, its items (q and k heads, runs of value channels, the gates) over the warps of `splits` blocks.
template <typename T, int V>
__device__ __forceinline__ void delta_prepare_token(const DeltaInputs& in, const T* __restrict__ proj, T* __restrict__ v_out, int token,
                                                    int item0, int step, int lane) {
    const int d = in.d, taps = in.taps, heads = in.heads, kv_heads = in.kv_heads, e = in.e;
    const int pos = in.positions[token], row = in.token_row[token];
    const int qk_width = kv_heads * d, channels = 2 * qk_width + heads * e;
    int history = 0;                 // how many earlier positions this step itself brought (at most taps - 1 matter)
    while (history < taps - 1 && token - history - 1 >= 0 && in.token_row[token - history - 1] == row
           && in.positions[token - history - 1] == pos - history - 1)
        ++history;
    const bool alone = history == 0 && (token + 1 >= in.n_tokens || in.token_row[token + 1] != row);
    float* slot = in.state + (size_t)row * (taps - 1) * channels;
    const T* mine = proj + (size_t)token * in.ld;
    auto convolved = [&](int c) {
        MsVec<V> y;
#pragma unroll
        for (int i = 0; i < V; ++i) y.x[i] = 0.f;
        for (int j = 0; j < taps; ++j) {
            const int back = taps - 1 - j;
            MsVec<V> u;
#pragma unroll
            for (int i = 0; i < V; ++i) u.x[i] = 0.f;
            if (back <= history) u = ms_read<T, V>(mine - (long long)back * in.ld + c);
            else if (pos - back >= 0) u = ms_read<float, V>(slot + (size_t)(taps - 1 - (back - history)) * channels + c);
            // row j of the slot is read before row j - 1 is overwritten by it, and by this thread alone
            if (alone && j > 0) ms_write(slot + (size_t)(j - 1) * channels + c, u);
            const MsVec<V> w = ms_read<float, V>(in.taps_w + (size_t)j * channels + c);
#pragma unroll
            for (int i = 0; i < V; ++i) y.x[i] = fmaf(w.x[i], u.x[i], y.x[i]);
        }
#pragma unroll
        for (int i = 0; i < V; ++i) y.x[i] = ms_silu(y.x[i]);
        return y;
    };
    const int v_items = (heads * e + 32 * V - 1) / (32 * V);
    float* qk_row = in.qk + (size_t)token * 2 * qk_width;
    for (int item = item0; item < 2 * kv_heads + v_items + 1; item += step) {
        if (item < 2 * kv_heads) {                      // a q or a k head
            const int c0 = item * d;
            const float scale = item < kv_heads ? in.q_scale : 1.f;
            MsVec<V> kept[MS_PREPARE_KEPT / V];
            float ss = 0.f;
            for (int n = 0, c = lane * V; c < d; ++n, c += 32 * V) {
                const MsVec<V> y = convolved(c0 + c);
#pragma unroll
                for (int i = 0; i < V; ++i) ss = fmaf(y.x[i], y.x[i], ss);
#pragma unroll
                for (int m = 0; m < MS_PREPARE_KEPT / V; ++m) if (m == n) kept[m] = y;
                if (n >= MS_PREPARE_KEPT / V) ms_write(qk_row + c0 + c, y);
            }
            ss = warp_sum(ss);
            const float inv = scale / sqrtf(ss + 1e-6f);
            for (int n = 0, c = lane * V; c < d; ++n, c += 32 * V) {
                MsVec<V> y;
                if (n >= MS_PREPARE_KEPT / V) y = ms_read<float, V>(qk_row + c0 + c);       // what this lane wrote above
#pragma unroll
                for (int m = 0; m < MS_PREPARE_KEPT / V; ++m) if (m == n) y = kept[m];
#pragma unroll
                for (int i = 0; i < V; ++i) y.x[i] *= inv;
                ms_write(qk_row + c0 + c, y);
            }
        } else if (item < 2 * kv_heads + v_items) {     // 32 * V value channels
            const int c = (item - 2 * kv_heads) * 32 * V + lane * V;
            if (c < heads * e) ms_write(v_out + (size_t)token * heads * e + c, convolved(2 * qk_width + c));
        } else {
            delta_gates<T>(in, mine, token, lane);
        }
    }
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const T* __restrict__ proj, DeltaInputs in, T* __restrict__ v_out) {
    qil_wait_for_producer();
    qil_release_consumer();
    delta_prepare_token<T, V>(in, proj, v_out, blockIdx.x, blockIdx.y * 8 + (threadIdx.x >> 5), 8 * gridDim.y, threadIdx.x & 31);
}

// Prompts: MS_RUN tokens a block.  Where they and the TAPS - 1 rows before them are one request's, a lane reads every row of its
// four channels once for all of them (heads of at most 128 channels); else token by token.  The same sums in the same order.
#define MS_RUN 4
template <typename T, int TAPS>
__global__ void __launch_bounds__(256)
delta_prepare_run_kernel(const T* __restrict__ proj, DeltaInputs in, T* __restrict__ v_out) {
    const int token0 = blockIdx.x * MS_RUN, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int before = token0 - (TAPS - 1), last = token0 + MS_RUN - 1;
    const bool whole = before >= 0 && last < in.n_tokens && in.token_row[before] == in.token_row[last]
                       && in.positions[last] - in.positions[before] == MS_RUN + TAPS - 2;
    qil_wait_for_producer();
    qil_release_consumer();
    if (!whole) {
        for (int token = token0; token <= min(last, in.n_tokens - 1); ++token)
            delta_prepare_token<T, 4>(in, proj, v_out, token, warp, 8, lane);
        return;
    }
    const int d = in.d, heads = in.heads, kv_heads = in.kv_heads, e = in.e;
    const int qk_width = kv_heads * d, channels = 2 * qk_width + heads * e, v_items = (heads * e + 127) / 128;
    const T* first_row = proj + (size_t)before * in.ld;
    for (int item = warp; item < 2 * kv_heads + v_items + MS_RUN; item += 8) {
        if (item >= 2 * kv_heads + v_items) {
            const int token = token0 + item - (2 * kv_heads + v_items);
            delta_gates<T>(in, proj + (size_t)token * in.ld, token, lane);
            continue;
        }
        const bool is_head = item < 2 * kv_heads;
        const int c = is_head ? item * d + lane * 4 : 2 * qk_width + (item - 2 * kv_heads) * 128 + lane * 4;
        const bool mine = is_head ? lane * 4 < d : c < channels;
        MsVec<4> u[MS_RUN + TAPS - 1], w[TAPS], y[MS_RUN];
#pragma unroll
        for (int i = 0; i < MS_RUN + TAPS - 1; ++i) u[i] = mine ? ms_read<T, 4>(first_row + (size_t)i * in.ld + c) : MsVec<4>{{0.f, 0.f, 0.f, 0.f}};
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = mine ? ms_read<float, 4>(in.taps_w + (size_t)j * channels + c) : MsVec<4>{{0.f, 0.f, 0.f, 0.f}};
        float ss[MS_RUN];
#pragma unroll
        for (int t = 0; t < MS_RUN; ++t) {
            ss[t] = 0.f;
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                float sum = 0.f;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) sum = fmaf(w[j].x[i], u[t + j].x[i], sum);
                y[t].x[i] = ms_silu(sum);
                ss[t] = fmaf(y[t].x[i], y[t].x[i], ss[t]);
            }
        }
        if (is_head) {
#pragma unroll
            for (int t = 0; t < MS_RUN; ++t) {
                const float inv = (item < kv_heads ? in.q_scale : 1.f) / sqrtf(warp_sum(ss[t]) + 1e-6f);
#pragma unroll
                for (int i = 0; i < 4; ++i) y[t].x[i] *= inv;
                if (mine) ms_write(in.qk + (size_t)(token0 + t) * 2 * qk_width + c, y[t]);
            }
        } else if (mine) {
#pragma unroll
            for (int t = 0; t < MS_RUN; ++t) ms_write(v_out + (size_t)(token0 + t) * heads * e + c - 2 * qk_width, y[t]);
        }
    }
}

extern "C" int qil_delta_prepare(const void* proj, long long ld, int b_col, int a_col, const float* taps_w, int taps, float* state,
                                 const float* a_log, const float* dt_bias, float q_scale, const int* positions,
                                 const int* token_row, int n_tokens, int heads, int kv_heads, int d, int e, float* qk, void* v_out,
                                 float* beta, float* log_decay, int act_dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || d <= 0 || e <= 0 || taps < 1)
        QIL_REFUSE("delta_prepare: heads %d/%d sizes %d/%d taps %d", heads, kv_heads, d, e, taps);
    if (taps > 1 && state == nullptr) QIL_REFUSE("delta_prepare: a convolution over time needs its state");
    const bool wide = d % 4 == 0 && (heads * e) % 4 == 0 && ld % 4 == 0 &&
                      (((uintptr_t)proj | (uintptr_t)taps_w | (uintptr_t)state | (uintptr_t)qk | (uintptr_t)v_out) & 15) == 0;
    const DeltaInputs in = {ld, b_col, a_col, taps_w, taps, state, a_log, dt_bias, q_scale, positions, token_row, n_tokens, heads,
                            kv_heads, d, e, qk, beta, log_decay};
    const int lanes = wide ? 4 : 1, items = 2 * kv_heads + (heads * e + 32 * lanes - 1) / (32 * lanes) + 1;
    int splits = 1;                 // few tokens (a decode step): a token's items over several blocks
    while (splits < 16 && (long long)n_tokens * splits < 148 && splits * 8 < items) splits <<= 1;
    const bool runs = wide && d <= 128 && taps >= 2 && taps <= 4 && n_tokens >= 16 * MS_RUN;
#define QIL_PREPARE_RUN(TAPS)                                                                                              \
    qil_launch_chained(delta_prepare_run_kernel<T, TAPS>, dim3((n_tokens + MS_RUN - 1) / MS_RUN), dim3(256), 0, stream,    \
                       (const T*)proj, in, (T*)v_out)
#define QIL_PREPARE_GO(V)                                                                                                  \
    qil_launch_chained(delta_prepare_kernel<T, V>, dim3(n_tokens, splits), dim3(256), 0, stream, (const T*)proj, in, (T*)v_out)
    QIL_DISPATCH_1(act_dtype, {
        if (runs) { if (taps == 2) QIL_PREPARE_RUN(2); else if (taps == 3) QIL_PREPARE_RUN(3); else QIL_PREPARE_RUN(4); }
        else if (wide) QIL_PREPARE_GO(4);
        else QIL_PREPARE_GO(1);
    });
#undef QIL_PREPARE_RUN
#undef QIL_PREPARE_GO
    QIL_CHECK_LAUNCH();
}

// Gated linear attention with a decay per key channel, as a scan over the tokens of every segment.
//
// Per head, with a state S [d, e] (d key channels, e value channels) kept in float32 per request:
//
//   a_t = sigmoid(z_t)^(1/tau),  z_t = A2 low_t + b           (float32; low_t is the low-rank projection;
//                                                             a kernel of its own, once per layer and step)
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T
//   o_t = S_t^T (q_t * q_scale)
//   y_t = o_t / sqrt(mean_e(o_t^2) + eps) * w  *  silu(g_t)   (norm over the head's e values, gate from a projection)
//
// One block owns one (segment, head, tile of value columns): a thread holds a slice of one or two columns of S in
// registers for the whole segment (two where one column a thread would not hold all of a head's values: what is read
// of q, k and the decays then serves both), reads the state slot of the segment's request at the start and writes
// it back at the end, so a prompt portion goes on from what the portions before it left, and a single
// decoded token is a segment of length one.  When one tile holds all of a head's value columns the norm
// and the gate are applied by the same block; otherwise o goes to a float32 scratch buffer and a row
// kernel norms and gates it.  Tokens are taken in their order with float32 arithmetic, so the
// result does not depend on how a sequence was cut into segments.  Tokens are staged in batches of
// GLA_TB: one barrier pair per batch instead of per token.
//
// Long segments are cut into chunks that run side by side (the `mode` of the entry point): mode 1 scans
// every chunk from a zero state and leaves the chunk's own state and the product of its decays; a carry
// kernel walks a segment's chunks in order, S_in(c+1) = P(c) S_in(c) + S_own(c), leaving every chunk's
// incoming state in place of its own and the last one in the request's slot; mode 2 scans every chunk
// again from its incoming state and writes the outputs.  Twice the arithmetic, all chunks at once.  The
// carry rounds differently from the token-by-token scan: results then depend on the cut in the last bits.
//
// q, k, v, g and low are column ranges of one row-major buffer (the stacked projection), given as
// pointers to their first column and the common row stride.
//
// Two options serve linear attention with a fixed decay per head, S_t = decay_h S_(t-1) + k_t v_t^T:
// `head_decay` (float32 [heads]) stands in for the per-token decays, and `qkv_act` 1 applies silu to q, k
// and v as they are read (in float32).  Such a design norms all heads' outputs together: `force_raw` sends
// the un-normed outputs to the float32 scratch buffer whatever the sizes, and lin_norm_gate_whole
// finishes them (one norm over a token's whole row, times sigmoid of the gate).
//
// Further forms of what enters the recurrence (`ScanInputs`; all of it float32):
//
//   tied gate      k holds a gate's logits z: f = l + (1 - l) sigmoid(z + b) per head and key channel (bias b and lower
//                  bound l, float or bfloat16 [heads * d]); the channel decays by f and is written with 1 - f, computed
//                  as (1 - l) sigmoid(-(z + b)) so that a gate near one loses nothing
//   token scalars  a decay and a write gain per token and head (float32 [tokens, heads], `mlstm_gates` makes them):
//                  S_t = decay S_(t-1) + gain k_t v_t^T
//   ones           the state has one column more than the values: its value is the constant one, so that the column
//                  is the sum of the decayed keys, n_t = decay n_(t-1) + gain k_t, and its output is n_t . q_t
//
// mlstm_gates walks the two gates of a matrix memory (log input gate i, log forget gate f, both capped by
// cap tanh(. / cap), the forget gate through a log sigmoid) over a segment's tokens from the running maximum m in the
// request's slot: m_t = max(f_t + m_(t-1), i_t), decay_t = exp(f_t + m_(t-1) - m_t), gain_t = exp(i_t - m_t),
// floor_t = exp(-m_t).  The maximum is a chain of single additions and comparisons in token order, the same bits under
// every cut.  With the floors the scan finishes the memory's outputs itself where a block holds all of a head's
// columns (o over max(|n . q|, floor) + 1e-6, over its own root mean square, times a weight per element of all heads and
// sigmoid of a gate); else mlstm_finish does, from the raw outputs.
#include "common.cuh"
#include "head_norm_gate.cuh"

#define GLA_TB 8

__device__ __forceinline__ float decay_from_logit(float z, float inv_tau) {
    // sigmoid(z)^(1/tau) = exp(log_sigmoid(z) / tau);  log_sigmoid(z) = min(z, 0) - log1p(exp(-|z|))
    const float log_sigmoid = fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
    return expf(log_sigmoid * inv_tau);
}

#define GLA_R 32          // rows of a column that one thread holds
#define GLA_THREADS 256
#ifndef GLA_LOADS_AHEAD
#define GLA_LOADS_AHEAD 2 // groups of four rows whose q, k and decays are on their way at a time
#endif
#define GLA_MOST_THREADS 288   // with a column of ones beside a full block of value columns
#ifndef GLA_MIN_BLOCKS
#define GLA_MIN_BLOCKS 2  // blocks per multiprocessor the scan is compiled for
#endif

// alpha[t, c] = sigmoid(b_c + sum_j A2[c, j] low[t, j])^(1/tau) for every token and key channel: float32, once
// per layer and step (the scan's blocks all read it).
template <typename T, typename W>
__global__ void __launch_bounds__(256)
gla_decay_kernel(const T* __restrict__ low, int ld, const W* __restrict__ a2, const W* __restrict__ a2_bias, int rank,
                 float inv_tau, int channels, float* __restrict__ alpha) {
    extern __shared__ float s_low[];        // [rank]
    qil_wait_for_producer();
    qil_release_consumer();
    const size_t token = blockIdx.x;
    for (int j = threadIdx.x; j < rank; j += 256) s_low[j] = to_f32<T>(low[token * ld + j]);
    __syncthreads();
    for (int c = threadIdx.x; c < channels; c += 256) {
        float z = to_f32<W>(a2_bias[c]);
        const W* a2_row = a2 + (size_t)c * rank;
        for (int j = 0; j < rank; ++j) z = fmaf(to_f32<W>(a2_row[j]), s_low[j], z);
        alpha[token * channels + c] = decay_from_logit(z, inv_tau);
    }
}

__device__ __forceinline__ float scan_input(float x, int act) { return act ? x / (1.f + expf(-x)) : x; }

// Where the decays come from, and what is done to q, k and v as they are read.
struct ScanInputs {
    const float* alpha;          // float32 [tokens, heads * d]: a decay per token and key channel
    const float* head_decay;     // float32 [heads]: one fixed decay per head
    const void* gate_bias;       // tied gate, in the weights' type [heads * d]: its bias ...
    const void* gate_lower;      // ... and its lower bound; k then holds the gate's logits
    const float* token_decay;    // float32 [tokens, heads]
    const float* token_gain;     // float32 [tokens, heads]
    const float* floor_;         // GLA_MEMORY: float32 [tokens, heads]
    int act;                     // bit 0: silu on q, bit 1: on k, bit 2: on v
    int ones;                    // 1: the state's last column has the constant value one
};
#define SCAN_SILU_Q 1
#define SCAN_SILU_K 2
#define SCAN_SILU_V 4

// What the block does with its outputs.
#define GLA_RAW 0          // float32 scratch, as they are
#define GLA_NORM 1         // normed per head, gated
#define GLA_MEMORY 2       // over max(|n . q|, floor) + 1e-6 (n . q is the last column), normed per head, weight, output gate

#define GLA_WHOLE 0        // from the state slot, outputs, state written back
#define GLA_OWN_STATE 1    // from zero, no outputs; the chunk's state and the product of its decays are written
#define GLA_FROM_STATE 2   // from the given state, outputs, nothing written back

#define MEMORY_ROW 4     // values of a head's row that a lane holds
// A matrix memory's outputs of one token and head: o over its size, over its own root mean square, weight, output gate.
template <typename T, typename W>
__device__ __forceinline__ void memory_finish_row(const float* o, int e, float floor_, const T* g, const W* norm_w, float eps,
                                                  T* out, int lane) {
    const float size = fmaxf(fabsf(o[e]), floor_) + 1e-6f;
    float ss = 0.f;
    if (e <= 32 * MEMORY_ROW) {           // everything is asked for before the first value is used
        float v[MEMORY_ROW], gate[MEMORY_ROW], w[MEMORY_ROW];
#pragma unroll
        for (int u = 0; u < MEMORY_ROW; ++u) {
            const int c = lane + 32 * u;
            v[u] = c < e ? o[c] : 0.f;
            gate[u] = c < e ? to_f32<T>(g[c]) : 0.f;
            w[u] = c < e ? to_f32<W>(norm_w[c]) : 0.f;
        }
#pragma unroll
        for (int u = 0; u < MEMORY_ROW; ++u) { v[u] = v[u] / size; ss = fmaf(v[u], v[u], ss); }
        ss = warp_sum(ss);
        const float scale = 1.0f / sqrtf(ss / (float)e + eps);
#pragma unroll
        for (int u = 0; u < MEMORY_ROW; ++u)
            if (lane + 32 * u < e) out[lane + 32 * u] = from_f32<T>(v[u] * scale * w[u] * (1.f / (1.f + expf(-gate[u]))));
        return;
    }
    for (int c = lane; c < e; c += 32) { const float v = o[c] / size; ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    const float scale = 1.0f / sqrtf(ss / (float)e + eps);
    for (int c = lane; c < e; c += 32) {
        const float gate = to_f32<T>(g[c]);
        out[c] = from_f32<T>(o[c] / size * scale * to_f32<W>(norm_w[c]) * (1.f / (1.f + expf(-gate))));
    }
}

// SCALAR: one decay per token (a head's own, or per token and head) for all key channels, in a register instead of a
// shared array.  CPT: value columns a thread holds.
template <typename T, typename W, int FUSE, int MODE, int CPT, bool SCALAR>
__global__ void __launch_bounds__(GLA_MOST_THREADS, GLA_MIN_BLOCKS)
gla_scan_kernel(const T* __restrict__ q, const T* __restrict__ k, const T* __restrict__ v, const T* __restrict__ g,
                ScanInputs in, int ld, float q_scale,
                const W* __restrict__ norm_w, float eps, float* __restrict__ state, float* __restrict__ decay_product, const int* __restrict__ seg_start,
                const int* __restrict__ seg_len, const int* __restrict__ seg_row, int n_heads, int d, int e,
                int ds_count, int tile_cols, float* __restrict__ o_raw, T* __restrict__ out) {
    constexpr int R = GLA_R;
    extern __shared__ float smem[];
    // q, k and the decays of a token: ds_count blocks of R values, each followed by four unused floats, so that
    // the threads of a quarter warp (which differ in their block) read their 16-byte pieces from different banks
    const int stride = ds_count * (R + 4);
    float* sq = smem;                    // [TB][stride]
    float* sk = sq + GLA_TB * stride;    // [TB][stride]
    float* sa = sk + GLA_TB * stride;    // [TB][stride], or with SCALAR [TB]
    float* sv = sa + (SCALAR ? GLA_TB : GLA_TB * stride);    // [TB][tile_cols]
    float* so = sv + GLA_TB * tile_cols; // [TB][tile_cols]
    float* sp = so + GLA_TB * tile_cols; // [d]: the product of the decays so far (GLA_OWN_STATE)
    qil_wait_for_producer();
    qil_release_consumer();
    const int tiles = (e + tile_cols - 1) / tile_cols;
    const int head = blockIdx.x / tiles, col0 = (blockIdx.x % tiles) * tile_cols, seg = blockIdx.y;
    const int first = seg_start[seg], count = seg_len[seg], row = seg_row[seg];
    const int tid = threadIdx.x, threads = blockDim.x;
    const int local = tid / ds_count, ds = tid % ds_count;
    const int half = (tile_cols + CPT - 1) / CPT;       // a thread's columns: local, local + half
    float* slot = state + ((size_t)row * n_heads + head) * d * e;

    bool owner[CPT];
    int at[CPT];
    float S[CPT][R];      // rows ds * R .. ds * R + R - 1 of the columns (rows past d stay zero)
#pragma unroll
    for (int j = 0; j < CPT; ++j) {
        at[j] = local + j * half;
        owner[j] = local < half && at[j] < tile_cols && col0 + at[j] < e;
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int dd = ds * R + r;
            S[j][r] = (MODE != GLA_OWN_STATE && owner[j] && dd < d) ? slot[(size_t)dd * e + col0 + at[j]] : 0.f;
        }
    }
    if (MODE == GLA_OWN_STATE)
        for (int dd = tid; dd < d; dd += threads) sp[dd] = 1.f;
    const int lane = tid & 31, warp = tid >> 5, warps = threads >> 5;
    const int values = e - in.ones;
    for (int t0 = 0; t0 < count; t0 += GLA_TB) {
        const int nb = count - t0 < GLA_TB ? count - t0 : GLA_TB;
        __syncthreads();
        for (int i = tid; i < nb * ds_count * R; i += threads) {
            const int tb = i / (ds_count * R), dd = i % (ds_count * R);
            const int to = tb * stride + (dd / R) * (R + 4) + dd % R;
            const bool real = dd < d;           // rows past d: zeros, which keep their (zero) state rows zero
            const size_t from = (size_t)(first + t0 + tb) * ld + head * d + dd;
            if (MODE != GLA_OWN_STATE) sq[to] = real ? scan_input(to_f32<T>(q[from]), in.act & SCAN_SILU_Q) * q_scale : 0.f;
            const float kv = real ? to_f32<T>(k[from]) : 0.f;
            float key = 0.f, decay = 0.f;
            if (real) {
                if (!SCALAR && in.gate_lower != nullptr) {
                    // both halves from one exponential of a negative number: sigmoid(z) and sigmoid(-z), neither by a
                    // difference from one
                    const float low = to_f32<W>(reinterpret_cast<const W*>(in.gate_lower)[head * d + dd]);
                    const float z = kv + to_f32<W>(reinterpret_cast<const W*>(in.gate_bias)[head * d + dd]);
                    const float small = expf(-fabsf(z)), inv = 1.f / (1.f + small);
                    const float up = z >= 0.f ? inv : small * inv, down = z >= 0.f ? small * inv : inv;
                    decay = fmaf(1.f - low, up, low);
                    key = (1.f - low) * down;
                } else {
                    key = scan_input(kv, in.act & SCAN_SILU_K);
                    if (SCALAR) {
                        if (in.token_gain != nullptr) key *= in.token_gain[(size_t)(first + t0 + tb) * n_heads + head];
                    } else {
                        decay = in.alpha[(size_t)(first + t0 + tb) * n_heads * d + head * d + dd];
                    }
                }
            }
            sk[to] = key;
            if (!SCALAR) sa[to] = decay;
        }
        if (SCALAR && tid < nb)
            sa[tid] = in.token_decay != nullptr ? in.token_decay[(size_t)(first + t0 + tid) * n_heads + head] : in.head_decay[head];
        for (int i = tid; i < nb * tile_cols; i += threads) {
            const int tb = i / tile_cols, c = col0 + i % tile_cols;
            sv[i] = c < values ? scan_input(to_f32<T>(v[(size_t)(first + t0 + tb) * ld + head * values + c]), in.act & SCAN_SILU_V)
                               : (c < e ? 1.f : 0.f);
        }
        __syncthreads();
        if (MODE == GLA_OWN_STATE) {
            for (int dd = tid; dd < d; dd += threads) {       // the same thread every batch: no barrier needed
                float product = sp[dd];
                for (int tb = 0; tb < nb; ++tb) product *= SCALAR ? sa[tb] : sa[tb * stride + (dd / R) * (R + 4) + dd % R];
                sp[dd] = product;
            }
        }
        for (int tb = 0; tb < nb; ++tb) {
            float vc[CPT], o[CPT];
#pragma unroll
            for (int j = 0; j < CPT; ++j) { vc[j] = owner[j] ? sv[tb * tile_cols + at[j]] : 0.f; o[j] = 0.f; }
            const float4* a4 = reinterpret_cast<const float4*>(sa + tb * stride + ds * (R + 4));
            const float4* k4 = reinterpret_cast<const float4*>(sk + tb * stride + ds * (R + 4));
            const float4* q4 = reinterpret_cast<const float4*>(sq + tb * stride + ds * (R + 4));
            const float scalar = SCALAR ? sa[tb] : 0.f;
#pragma unroll
            for (int r4 = 0; r4 < R / 4; ++r4) {
                // two columns of state fill the registers: shared loads must not all be moved to the front
                if (CPT > 1 && r4 > 0 && r4 % GLA_LOADS_AHEAD == 0) asm volatile("" ::: "memory");
                const float4 a = SCALAR ? make_float4(scalar, scalar, scalar, scalar) : a4[r4], kk = k4[r4];
                const float4 qq = MODE != GLA_OWN_STATE ? q4[r4] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int j = 0; j < CPT; ++j) {
                    S[j][4 * r4 + 0] = fmaf(a.x, S[j][4 * r4 + 0], kk.x * vc[j]);
                    S[j][4 * r4 + 1] = fmaf(a.y, S[j][4 * r4 + 1], kk.y * vc[j]);
                    S[j][4 * r4 + 2] = fmaf(a.z, S[j][4 * r4 + 2], kk.z * vc[j]);
                    S[j][4 * r4 + 3] = fmaf(a.w, S[j][4 * r4 + 3], kk.w * vc[j]);
                    if (MODE != GLA_OWN_STATE) {
                        o[j] = fmaf(S[j][4 * r4 + 0], qq.x, o[j]);
                        o[j] = fmaf(S[j][4 * r4 + 1], qq.y, o[j]);
                        o[j] = fmaf(S[j][4 * r4 + 2], qq.z, o[j]);
                        o[j] = fmaf(S[j][4 * r4 + 3], qq.w, o[j]);
                    }
                }
            }
            if (MODE == GLA_OWN_STATE) continue;
#pragma unroll
            for (int j = 0; j < CPT; ++j) {
                for (int step = 1; step < ds_count; step <<= 1) o[j] += __shfl_xor_sync(0xffffffffu, o[j], step);
                if (owner[j] && ds == 0) {
                    if (FUSE != GLA_RAW) so[tb * tile_cols + at[j]] = o[j];
                    else o_raw[((size_t)(first + t0 + tb) * n_heads + head) * e + col0 + at[j]] = o[j];
                }
            }
        }
        if (FUSE == GLA_NORM && MODE != GLA_OWN_STATE) {
            __syncthreads();
            head_norm_gate_rows<T, W>(so, tile_cols, nb, (size_t)(first + t0), g, ld, norm_w, eps, n_heads, head, e, out,
                                     lane, warp, warps);
        }
        if (FUSE == GLA_MEMORY && MODE != GLA_OWN_STATE) {
            __syncthreads();
            for (int tb = warp; tb < nb; tb += warps) {
                const size_t token = first + t0 + tb, pair = token * n_heads + head;
                memory_finish_row<T, W>(so + tb * tile_cols, values, in.floor_[pair], g + token * ld + head * values,
                                        norm_w + head * values, eps, out + pair * values, lane);
            }
        }
    }
    if (MODE == GLA_FROM_STATE) return;
    int pitch = e;
    asm volatile("" : "+r"(pitch));        // the addresses of the loads at the top must not be kept until here
#pragma unroll
    for (int j = 0; j < CPT; ++j)
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int dd = ds * R + r;
            if (owner[j] && dd < d) slot[(size_t)dd * pitch + col0 + at[j]] = S[j][r];
        }
    if (MODE == GLA_OWN_STATE && col0 == 0)
        for (int dd = tid; dd < d; dd += threads) decay_product[((size_t)row * n_heads + head) * d + dd] = sp[dd];
}

// The carry over a long segment's chunks: chunk_state [chunks, heads, d, e] holds every chunk's own state on
// entry and its incoming state on exit; the state after the last chunk goes to the request's slot.
// carry: int32 [n, 3] = (state slot, first chunk, chunks).
#define GLA_CARRY_AHEAD 16
__global__ void __launch_bounds__(256)
gla_carry_kernel(float* __restrict__ chunk_state, const float* __restrict__ decay_product, float* __restrict__ slots,
                 const int* __restrict__ carry, int n_heads, int d, int e) {
    qil_wait_for_producer();
    qil_release_consumer();
    const size_t per_state = (size_t)n_heads * d * e;
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x;
    if (i >= per_state) return;
    const int row = carry[3 * blockIdx.y], first = carry[3 * blockIdx.y + 1], chunks = carry[3 * blockIdx.y + 2];
    const size_t channel = i / e;                 // head * d + key channel
    float s = slots[(size_t)row * per_state + i];
    // GLA_CARRY_AHEAD chunks at a time: their loads are all under way before the first is used (a thread reads and writes
    // only its own element of every chunk, so the order of loads and stores between chunks is free)
    for (int c0 = first; c0 < first + chunks; c0 += GLA_CARRY_AHEAD) {
        float own[GLA_CARRY_AHEAD], decay[GLA_CARRY_AHEAD];
#pragma unroll
        for (int u = 0; u < GLA_CARRY_AHEAD; ++u) {
            const bool real = c0 + u < first + chunks;
            own[u] = real ? chunk_state[(size_t)(c0 + u) * per_state + i] : 0.f;
            decay[u] = real ? decay_product[(size_t)(c0 + u) * n_heads * d + channel] : 1.f;
        }
#pragma unroll
        for (int u = 0; u < GLA_CARRY_AHEAD; ++u) {
            if (c0 + u >= first + chunks) break;
            chunk_state[(size_t)(c0 + u) * per_state + i] = s;
            s = fmaf(decay[u], s, own[u]);
        }
    }
    slots[(size_t)row * per_state + i] = s;
}

// The norm and the gate for heads whose value columns were spread over several blocks: one block per token.
template <typename T, typename W>
__global__ void __launch_bounds__(256)
gla_norm_gate_kernel(const float* __restrict__ o_raw, const T* __restrict__ g, int ld, const W* __restrict__ norm_w,
                     float eps, int n_heads, int e, T* __restrict__ out) {
    qil_wait_for_producer();
    qil_release_consumer();
    const size_t token = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    for (int head = warp; head < n_heads; head += 8)
        head_norm_gate_rows<T, W>(o_raw + (token * n_heads + head) * e, 0, 1, token, g, ld, norm_w, eps, n_heads, head, e,
                                 out, lane, 0, 1);
}

struct ScanShape { int ds_count, tile_cols, tiles, threads, columns_a_thread; size_t smem; };

// A thread holds GLA_R rows of a column; ds_count threads (a power of two within a warp) share a column.  One column a
// thread where that holds all of a head's values in a block, else two for the chunks of long portions (there are blocks
// enough, and what is read of q, k and the decays serves both columns) and one for short segments from slot to slot,
// single tokens above all, where more blocks fetch the states sooner.
static bool scan_shape(int d, int e, int ones, bool scalar, bool whole, ScanShape& s) {
    s.ds_count = 1;
    while (s.ds_count * GLA_R < d) s.ds_count <<= 1;
    if (s.ds_count > 32) return false;
    s.columns_a_thread = (whole || e <= GLA_THREADS / s.ds_count) ? 1 : 2;
    const int most = s.columns_a_thread * (GLA_THREADS / s.ds_count);
    // a column of ones beside a full block of values takes one more warp, not one more block
    s.tiles = (ones && s.ds_count <= 32 && e == most + 1) ? 1 : (e + most - 1) / most;
    s.tile_cols = (e + s.tiles - 1) / s.tiles;             // even tiles
    s.threads = ((s.tile_cols + s.columns_a_thread - 1) / s.columns_a_thread * s.ds_count + 31) / 32 * 32;
    const int stride = s.ds_count * (GLA_R + 4);
    s.smem = ((size_t)GLA_TB * ((scalar ? 2 : 3) * stride + (scalar ? 1 : 0) + 2 * s.tile_cols) + d) * sizeof(float);
    return s.threads <= GLA_MOST_THREADS;
}

template <typename T, typename W, int FUSE, int MODE, int CPT, bool SCALAR>
static cudaError_t gla_launch(dim3 grid, const ScanShape& s, cudaStream_t stream, const void* q, const void* k,
                              const void* v, const void* g, ScanInputs in, int ld, float q_scale, const void* norm_w, float eps, float* state,
                              float* decay_product, const int* seg_start, const int* seg_len, const int* seg_row, int n_heads, int d, int e,
                              float* o_raw, void* out) {
    cudaError_t err = cudaFuncSetAttribute(gla_scan_kernel<T, W, FUSE, MODE, CPT, SCALAR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s.smem);
    if (err != cudaSuccess) return err;
    return qil_launch_chained(gla_scan_kernel<T, W, FUSE, MODE, CPT, SCALAR>, grid, dim3(s.threads), s.smem, stream,
                              (const T*)q, (const T*)k, (const T*)v, (const T*)g, in, ld, q_scale,
                              (const W*)norm_w, eps, state, decay_product, seg_start, seg_len, seg_row, n_heads, d, e,
                              s.ds_count, s.tile_cols, o_raw, (T*)out);
}

// o_raw: float32 [tokens, heads * e] of scratch, needed only when a head's value columns do not fit one
// block (qil_gla_scan_needs_scratch; e counts a column of ones; whole: for GLA_WHOLE, else for the chunks' modes).
extern "C" int qil_gla_scan_needs_scratch(int d, int e, int ones, int whole) {
    ScanShape s;
    if (!scan_shape(d, e, ones, false, whole != 0, s)) return -1;
    return s.tiles > 1 ? 1 : 0;
}

extern "C" int qil_gla_scan(const void* q, const void* k, const void* v, const void* g, const float* alpha,
                            const float* head_decay, const void* gate_bias, const void* gate_lower, const float* token_decay,
                            const float* token_gain, const float* floor_, int act, int ones, int force_raw, int ld, float q_scale, const void* norm_w, float eps, float* state, const int* seg_start, const int* seg_len,
                            const int* seg_row, int n_segments, int n_tokens, int n_heads, int d, int e, float* o_raw,
                            void* out, int mode, float* decay_product, int act_dtype, int weight_dtype,
                            cudaStream_t stream) {
    // mode: GLA_WHOLE; GLA_OWN_STATE (state: the chunks' states, seg_row: the chunk's index there, decay_product
    // [chunks, heads, d]); GLA_FROM_STATE (state and seg_row as before; the states are read only)
    if (n_segments <= 0) return 0;
    if (mode < 0 || mode > 2 || (mode == GLA_OWN_STATE && decay_product == nullptr)) QIL_REFUSE("gla_scan: mode %d", mode);
    const int sources = (alpha != nullptr) + (head_decay != nullptr) + (gate_lower != nullptr) + (token_decay != nullptr);
    if (sources != 1 || (gate_lower == nullptr) != (gate_bias == nullptr) || (token_decay == nullptr) != (token_gain == nullptr))
        QIL_REFUSE("gla_scan: exactly one source of decays, a gate with its bias, token decays with their gains");
    if (ones != 0 && (ones != 1 || e < 2)) QIL_REFUSE("gla_scan: a column of ones goes with values beside it");
    if (floor_ != nullptr && (ones != 1 || token_decay == nullptr || g == nullptr || norm_w == nullptr || out == nullptr))
        QIL_REFUSE("gla_scan: a matrix memory has a column of ones, token decays, an output gate and a norm");
    if (ones != 0 && floor_ == nullptr && !force_raw) QIL_REFUSE("gla_scan: a column of ones without a floor gives raw outputs");
    if (n_heads <= 0 || d <= 0 || e <= 0 || n_segments > 65535)
        QIL_REFUSE("gla_scan: heads %d sizes %d/%d segments %d", n_heads, d, e, n_segments);
    const bool scalar = head_decay != nullptr || token_decay != nullptr;
    ScanShape shape;
    if (!scan_shape(d, e, ones, scalar, mode == GLA_WHOLE, shape)) QIL_REFUSE("gla_scan: %d key channels per head are more than %d", d, 32 * GLA_R);
    const ScanInputs in = {alpha, head_decay, gate_bias, gate_lower, token_decay, token_gain, floor_, act, ones};
    const int fuse = (shape.tiles > 1 || force_raw) ? GLA_RAW : floor_ != nullptr ? GLA_MEMORY : GLA_NORM;
    if (fuse == GLA_NORM && scalar) QIL_REFUSE("gla_scan: one decay for all channels of a head goes with raw outputs or a matrix memory");
    if ((act_dtype != QIL_F32 && act_dtype != QIL_BF16) || (weight_dtype != QIL_F32 && (weight_dtype != QIL_BF16 || act_dtype == QIL_F32)))
        QIL_REFUSE("gla_scan: dtype codes %d/%d (float32 activations go with float32 parameters)", act_dtype, weight_dtype);
    if (fuse == GLA_RAW && o_raw == nullptr && mode != GLA_OWN_STATE) QIL_REFUSE("gla_scan: %d value columns per head need the scratch buffer", e);
    dim3 grid(n_heads * shape.tiles, n_segments);
    cudaError_t err = cudaSuccess;
#define QIL_GLA_RUN(T, W, F, M, C, S)                                                                              \
    (err = gla_launch<T, W, F, M, C, S>(grid, shape, stream, q, k, v, g, in, ld, q_scale, norm_w, eps, state,      \
                                        decay_product, seg_start, seg_len, seg_row, n_heads, d, e, o_raw, out))
#define QIL_GLA_GO(F, M, C, S)                                                                                     \
    do {                                                                                                           \
        if (act_dtype == QIL_F32) QIL_GLA_RUN(float, float, F, M, C, S);                                           \
        else if (weight_dtype == QIL_F32) QIL_GLA_RUN(bf16, float, F, M, C, S);                                    \
        else QIL_GLA_RUN(bf16, bf16, F, M, C, S);                                                                  \
    } while (0)
#define QIL_GLA_ONE(F, M, S) QIL_GLA_GO(F, M, 1, S)
#define QIL_GLA_COLS(F, M, S) do { if (shape.columns_a_thread == 1) QIL_GLA_GO(F, M, 1, S); else QIL_GLA_GO(F, M, 2, S); } while (0)
    // a memory's decays are scalars; a per-head norm goes with decays per channel
#define QIL_GLA_FUSE(M, COLS)                                                                                      \
    do {                                                                                                           \
        if (fuse == GLA_MEMORY) COLS(GLA_MEMORY, M, true);                                                         \
        else if (fuse == GLA_NORM) COLS(GLA_NORM, M, false);                                                       \
        else if (scalar) COLS(GLA_RAW, M, true);                                                                   \
        else COLS(GLA_RAW, M, false);                                                                              \
    } while (0)
    if (mode == GLA_OWN_STATE) { if (scalar) QIL_GLA_COLS(GLA_RAW, GLA_OWN_STATE, true); else QIL_GLA_COLS(GLA_RAW, GLA_OWN_STATE, false); }
    else if (mode == GLA_WHOLE) QIL_GLA_FUSE(GLA_WHOLE, QIL_GLA_ONE);
    else QIL_GLA_FUSE(GLA_FROM_STATE, QIL_GLA_COLS);
#undef QIL_GLA_FUSE
#undef QIL_GLA_COLS
#undef QIL_GLA_ONE
#undef QIL_GLA_GO
#undef QIL_GLA_RUN
    if (err != cudaSuccess) { snprintf(qil_error_text, sizeof(qil_error_text), "%s", cudaGetErrorString(err)); return (int)err; }
    QIL_CHECK_LAUNCH();
}

extern "C" int qil_gla_carry(float* chunk_state, const float* decay_product, float* slots, const int* carry,
                             int n_carries, int n_heads, int d, int e, cudaStream_t stream) {
    if (n_carries <= 0) return 0;
    const size_t per_state = (size_t)n_heads * d * e;
    qil_launch_chained(gla_carry_kernel, dim3((unsigned)((per_state + 255) / 256), n_carries), dim3(256), 0, stream,
                       chunk_state, (const float*)decay_product, slots, carry, n_heads, d, e);
    QIL_CHECK_LAUNCH();
}

// The norm and the gate over o_raw (what qil_gla_scan leaves when a head's value columns do not fit one block),
// once per step after all scans of the layer.
extern "C" int qil_gla_norm_gate(const float* o_raw, const void* g, int ld, const void* norm_w, float eps, int n_tokens,
                                 int n_heads, int e, void* out, int act_dtype, int weight_dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    QIL_DISPATCH_2(act_dtype, weight_dtype,
        qil_launch_chained(gla_norm_gate_kernel<T, W>, dim3(n_tokens), dim3(256), 0, stream, o_raw, (const T*)g, ld,
                           (const W*)norm_w, eps, n_heads, e, (T*)out));
    QIL_CHECK_LAUNCH();
}

// alpha float32 [n_tokens, channels] from the low-rank projection (columns of a row-major buffer of stride ld).
extern "C" int qil_gla_decay(const void* low, int ld, const void* a2, const void* a2_bias, int rank, float tau,
                             int n_tokens, int channels, float* alpha, int act_dtype, int weight_dtype,
                             cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rank <= 0 || channels <= 0 || !(tau > 0.f) || rank > 8192) QIL_REFUSE("gla_decay: rank %d channels %d tau %g", rank, channels, (double)tau);
    QIL_DISPATCH_2(act_dtype, weight_dtype,
        qil_launch_chained(gla_decay_kernel<T, W>, dim3(n_tokens), dim3(256), rank * sizeof(float), stream, (const T*)low, ld,
                           (const W*)a2, (const W*)a2_bias, rank, 1.f / tau, channels, alpha));
    QIL_CHECK_LAUNCH();
}

// out[n][i] = o_raw[n][i] / sqrt(mean_i(o_raw[n]^2) + eps) * w[i] * sigmoid(g[n][i]) over a token's whole row of
// `width` = heads * e values: the finish of a linear attention whose heads are normed together.
template <typename T, typename W>
__global__ void __launch_bounds__(256)
lin_norm_gate_whole_kernel(const float* __restrict__ o_raw, const T* __restrict__ g, int ld, const W* __restrict__ norm_w,
                           float eps, int width, T* __restrict__ out) {
    __shared__ float scratch[32];
    qil_wait_for_producer();
    qil_release_consumer();
    const size_t token = blockIdx.x;
    const float* o = o_raw + token * width;
    float ss = 0.f;
    for (int i = threadIdx.x; i < width; i += 256) ss = fmaf(o[i], o[i], ss);
    ss = block_sum(ss, scratch);
    const float scale = 1.0f / sqrtf(ss / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += 256) {
        const float gate = to_f32<T>(g[token * ld + i]);
        out[token * width + i] = from_f32<T>(o[i] * scale * to_f32<W>(norm_w[i]) * (1.f / (1.f + expf(-gate))));
    }
}

extern "C" int qil_lin_norm_gate_whole(const float* o_raw, const void* g, int ld, const void* norm_w, float eps,
                                       int n_tokens, int width, void* out, int act_dtype, int weight_dtype,
                                       cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (width <= 0) QIL_REFUSE("lin_norm_gate_whole: width %d", width);
    QIL_DISPATCH_2(act_dtype, weight_dtype,
        qil_launch_chained(lin_norm_gate_whole_kernel<T, W>, dim3(n_tokens), dim3(256), 0, stream, o_raw, (const T*)g, ld,
                           (const W*)norm_w, eps, width, (T*)out));
    QIL_CHECK_LAUNCH();
}

// ------------------------------------------------------------------ matrix memory: gates and finish
// One block per (segment, head).  igate, fgate: the gates' columns of the projection (head h at column h), row stride ld.
// m_slots float32 [slots, heads].  decay, gain, floor_ float32 [tokens, heads].  The gates of GATES_TOKENS tokens are made
// side by side, one thread walks their maximum, the exponentials are side by side again.
#define GATES_TOKENS 1024
template <typename T, typename W>
__global__ void __launch_bounds__(128)
mlstm_gates_kernel(const T* __restrict__ igate, const T* __restrict__ fgate, int ld, const W* __restrict__ i_bias,
                   const W* __restrict__ f_bias, float cap, float* __restrict__ m_slots, const int* __restrict__ seg_start,
                   const int* __restrict__ seg_len, const int* __restrict__ seg_row, int n_heads, float* __restrict__ decay,
                   float* __restrict__ gain, float* __restrict__ floor_) {
    __shared__ float2 gates[GATES_TOKENS];           // (log forget gate, log input gate)
    __shared__ float after[GATES_TOKENS + 1];        // the maximum before the first token and after each
    qil_wait_for_producer();
    qil_release_consumer();
    const int tid = threadIdx.x, head = blockIdx.x, seg = blockIdx.y;
    const int first = seg_start[seg], count = seg_len[seg], row = seg_row[seg];
    const float bi = to_f32<W>(i_bias[head]), bf = to_f32<W>(f_bias[head]);
    if (tid == 0) after[0] = m_slots[(size_t)row * n_heads + head];
    for (int t0 = 0; t0 < count; t0 += GATES_TOKENS) {
        const int nb = count - t0 < GATES_TOKENS ? count - t0 : GATES_TOKENS;
        for (int j = tid; j < nb; j += 128) {
            const size_t at = (size_t)(first + t0 + j) * ld + head;
            const float il = cap * tanhf((to_f32<T>(igate[at]) + bi) / cap);
            const float z = cap * tanhf((to_f32<T>(fgate[at]) + bf) / cap);
            gates[j] = make_float2(fminf(z, 0.f) - log1pf(expf(-fabsf(z))), il);
        }
        __syncthreads();
        if (tid == 0) {
            // sixteen tokens' gates are read before their maxima are written: a load does not wait for the store before it
            float m = after[0];
            int j = 0;
            for (; j + 16 <= nb; j += 16) {
                float2 g[16];
                float now[16];
#pragma unroll
                for (int u = 0; u < 16; ++u) g[u] = gates[j + u];
#pragma unroll
                for (int u = 0; u < 16; ++u) { m = fmaxf(g[u].x + m, g[u].y); now[u] = m; }
#pragma unroll
                for (int u = 0; u < 16; ++u) after[j + u + 1] = now[u];
            }
            for (; j < nb; ++j) {
                m = fmaxf(gates[j].x + m, gates[j].y);
                after[j + 1] = m;
            }
        }
        __syncthreads();
        for (int j = tid; j < nb; j += 128) {
            const float2 g = gates[j];
            const float before = after[j], now = after[j + 1];
            const size_t at = (size_t)(first + t0 + j) * n_heads + head;
            decay[at] = expf(g.x + before - now);
            gain[at] = expf(g.y - now);
            floor_[at] = expf(-now);
        }
        __syncthreads();
        if (tid == 0) after[0] = after[nb];
    }
    if (tid == 0) m_slots[(size_t)row * n_heads + head] = after[0];
}

extern "C" int qil_mlstm_gates(const void* igate, const void* fgate, int ld, const void* i_bias, const void* f_bias, float cap,
                               float* m_slots, const int* seg_start, const int* seg_len, const int* seg_row, int n_segments,
                               int n_heads, float* decay, float* gain, float* floor_, int act_dtype, int weight_dtype,
                               cudaStream_t stream) {
    if (n_segments <= 0) return 0;
    if (n_heads <= 0 || !(cap > 0.f) || n_segments > 65535) QIL_REFUSE("mlstm_gates: heads %d cap %g segments %d", n_heads, (double)cap, n_segments);
    QIL_DISPATCH_2(act_dtype, weight_dtype,
        qil_launch_chained(mlstm_gates_kernel<T, W>, dim3(n_heads, n_segments), dim3(128), 0, stream, (const T*)igate,
                           (const T*)fgate, ld, (const W*)i_bias, (const W*)f_bias, cap, m_slots, seg_start, seg_len, seg_row,
                           n_heads, decay, gain, floor_));
    QIL_CHECK_LAUNCH();
}

// raw float32 [tokens, heads, e + 1]: a head's e outputs and n . q behind them.  A warp per (token, head).
template <typename T, typename W>
__global__ void __launch_bounds__(256)
mlstm_finish_kernel(const float* __restrict__ raw, const float* __restrict__ floor_, const T* __restrict__ g, int ld,
                    const W* __restrict__ norm_w, float eps, int n_pairs, int n_heads, int e, T* __restrict__ out) {
    qil_wait_for_producer();
    qil_release_consumer();
    const int lane = threadIdx.x & 31;
    const size_t pair = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (pair >= (size_t)n_pairs) return;
    const size_t token = pair / n_heads;
    const int head = (int)(pair % n_heads);
    memory_finish_row<T, W>(raw + pair * (e + 1), e, floor_[pair], g + token * ld + head * e, norm_w + head * e, eps, out + pair * e, lane);
}

extern "C" int qil_mlstm_finish(const float* raw, const float* floor_, const void* g, int ld, const void* norm_w, float eps,
                                int n_tokens, int n_heads, int e, void* out, int act_dtype, int weight_dtype,
                                cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (n_heads <= 0 || e <= 0 || (long long)n_tokens * n_heads > 2000000000ll) QIL_REFUSE("mlstm_finish: heads %d values %d", n_heads, e);
    const int n_pairs = n_tokens * n_heads;
    QIL_DISPATCH_2(act_dtype, weight_dtype,
        qil_launch_chained(mlstm_finish_kernel<T, W>, dim3((n_pairs + 7) / 8), dim3(256), 0, stream, raw, floor_, (const T*)g, ld,
                           (const W*)norm_w, eps, n_pairs, n_heads, e, (T*)out));
    QIL_CHECK_LAUNCH();
}

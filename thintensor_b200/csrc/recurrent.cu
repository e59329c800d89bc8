// Kernels of the recurrent token mixers: the short causal convolution with its carried inputs, the
// Mamba-2 state-space recurrence (also run with a constant decay and step size one: the linear
// attention S <- g S + k v^T, o = S^T q, whose q, k and v a kernel here prepares), the gated delta-rule
// recurrence, both also with a decay of its own for every head and state row at every token, the products of low rank
// that such decays (and gates) come from, the gated group norm behind them (gate: silu or sigmoid), and the weighted sum of two branches.  Everything here is float32: inputs are the float32 partial
// sums of a projection ([splits][tokens][cols], summed on the way in), states live in float32 and are
// carried per sequence slot, and only the normalised output that feeds the next matrix product is
// narrowed to the activation dtype.
//
// Packed batches: token t belongs to the sequence b with cu[b] <= t < cu[b + 1]; its state lies at
// slots[b].  A recurrence walks a sequence's tokens in order and starts from the slot's state, so a
// prompt cut into steps, a prompt and its decoded tokens, and a sequence inside a batch all run the
// same chain of operations and give the same bits.
//
// A state matrix is owned column by column: the column of value dimension p (all its N state rows)
// belongs to a group of REC_LANES neighbouring lanes, lane l holding rows 4l .. 4l + 3, 4l + 32 .. 4l + 35, ...
// in registers (four neighbouring rows at a time, so that a token's vectors come out of shared memory, and the
// state out of global memory, in 16-byte pieces that the group's lanes read side by side).  Row products with the token's vectors (read from shared memory, where a chunk of tokens
// is staged) are summed inside the group with shuffles.  Columns are independent, so a CTA takes
// REC_COLS of them for one (sequence, head) and the grid is heads x sequences x column tiles.  When that
// grid would fill the GPU more than twice over, a lane group owns four neighbouring columns instead and
// a CTA 64 of them (see the kernels' template parameters).
#include "common.cuh"

constexpr int REC_LANES = 8;        // lanes that share one state column (measured on a B200, 64 heads of 64 x 128: one sequence of 2,048
                                    // tokens 0.79 ms with 8 lanes and 0.86 ms with 16; one token of 64 sequences 70 us and 94 us)
constexpr int REC_COLS = 32;        // state columns of a CTA (REC_COLS * REC_LANES threads)
constexpr int REC_CHUNK = 16;       // tokens staged in shared memory at a time
constexpr int REC_MAX_ROWS = 256;   // largest state size per column (N of Mamba-2, key size of the delta rule)
constexpr int CONV_MAX_TAPS = 8;

// sum of one element over the k-slices of a projection: four loads in flight together, additions in slice order
__device__ __forceinline__ float rec_sum_slices(const float* __restrict__ p, int splits, size_t split_stride) {
    float total = 0.0f;
    int s = 0;
    for (; s + 4 <= splits; s += 4) {
        const float a = __ldg(p + (size_t)s * split_stride), b = __ldg(p + (size_t)(s + 1) * split_stride);
        const float c = __ldg(p + (size_t)(s + 2) * split_stride), d = __ldg(p + (size_t)(s + 3) * split_stride);
        total = (((total + a) + b) + c) + d;
    }
    for (; s < splits; ++s) total += __ldg(p + (size_t)s * split_stride);
    return total;
}

// Asynchronous copies into shared memory: a chunk of tokens is fetched while the chunk before it is worked on.
__device__ __forceinline__ uint32_t rec_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void rec_copy4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(rec_smem(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void rec_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(rec_smem(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void rec_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void rec_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// rows x width floats from src (row stride src_stride) to dst (row stride dst_stride), all threads of the block taking
// part; vec: every row start and the width are multiples of four floats and both bases are 16-byte aligned
__device__ __forceinline__ void rec_stage(float* dst, int dst_stride, const float* src, size_t src_stride, int rows, int width, bool vec) {
    if (vec) {
        const int quads = width >> 2;
        for (int e = threadIdx.x; e < rows * quads; e += blockDim.x) {
            const int k = e / quads, r = (e - k * quads) << 2;
            rec_copy16(dst + k * dst_stride + r, src + (size_t)k * src_stride + r);
        }
    } else {
        for (int e = threadIdx.x; e < rows * width; e += blockDim.x) {
            const int k = e / width, r = e - k * width;
            rec_copy4(dst + k * dst_stride + r, src + (size_t)k * src_stride + r);
        }
    }
}

__device__ __forceinline__ float rec_silu(float x) { return x / (1.0f + expf(-x)); }
// the gate of a normed read-out: 0 silu, 1 sigmoid
__device__ __forceinline__ float rec_gate(float x, int kind) { return kind == 1 ? 1.0f / (1.0f + expf(-x)) : rec_silu(x); }
__device__ __forceinline__ float rec_softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

// the state row that register i of lane `lane` holds
__device__ __forceinline__ int rec_row(int lane, int i) { return 4 * lane + 4 * REC_LANES * (i >> 2) + (i & 3); }

// a column's registers from / to its N numbers in global memory
template <int K>
__device__ __forceinline__ void rec_load_column(float (&s)[K], const float* __restrict__ S, int lane, int N, bool live) {
#pragma unroll
    for (int j = 0; j < K / 4; ++j) {
        const int r = rec_row(lane, 4 * j);
        if (live && !(N & 3) && r < N) {
            const float4 v = *reinterpret_cast<const float4*>(S + r);
            s[4 * j] = v.x; s[4 * j + 1] = v.y; s[4 * j + 2] = v.z; s[4 * j + 3] = v.w;
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) s[4 * j + e] = (live && r + e < N) ? S[r + e] : 0.0f;
        }
    }
}
template <int K>
__device__ __forceinline__ void rec_store_column(const float (&s)[K], float* __restrict__ S, int lane, int N) {
#pragma unroll
    for (int j = 0; j < K / 4; ++j) {
        const int r = rec_row(lane, 4 * j);
        if (!(N & 3) && r < N) {
            *reinterpret_cast<float4*>(S + r) = make_float4(s[4 * j], s[4 * j + 1], s[4 * j + 2], s[4 * j + 3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (r + e < N) S[r + e] = s[4 * j + e];
        }
    }
}

// a token's vector (K * REC_LANES numbers in shared memory, zero beyond the real ones) into the registers that match the column's
template <int K>
__device__ __forceinline__ void rec_load_vector(float (&v)[K], const float* __restrict__ row, int lane) {
    const float4* row4 = reinterpret_cast<const float4*>(row);
#pragma unroll
    for (int j = 0; j < K / 4; ++j) {
        const float4 q = row4[lane + REC_LANES * j];
        v[4 * j] = q.x; v[4 * j + 1] = q.y; v[4 * j + 2] = q.z; v[4 * j + 3] = q.w;
    }
}

__device__ __forceinline__ float rec_group_sum(float v) {
#pragma unroll
    for (int o = REC_LANES / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// ------------------------------------------------------------------------------------
// Causal convolution over time, one filter per channel:
//   y[t, c] = f(bias[c] + sum_j w[c, j] * x[t - (taps - 1) + j, c]),   f = silu or identity.
// x before this step's first token comes from the sequence's state, which holds its last taps - 1
// inputs (oldest first, [taps - 1][channels]; zero for a new sequence).
// Prompts: one kernel computes the outputs, a second one moves the states on (a thread per sequence
// and channel), because the outputs of a sequence's first tokens read the state that the update
// overwrites.  One token per sequence: a thread per (sequence, channel) does both.
// ------------------------------------------------------------------------------------
constexpr int CONV_TILE = 16;       // packed tokens a thread walks with its channel's last inputs in registers

// A thread takes one channel through CONV_TILE packed tokens: every input is read once (plus taps - 1 at the tile's
// start) and the window of the last inputs slides through registers.  Where the tile crosses into the next sequence
// the window is filled from that sequence's state.
__global__ void causal_conv_kernel(const float* __restrict__ proj, int splits, size_t split_stride, int cols, int col_off,
                                   int channels, const float* __restrict__ weight, const float* __restrict__ bias, int taps,
                                   int activation, const float* __restrict__ state, size_t slot_stride, float* __restrict__ out,
                                   const int* __restrict__ cu, const int* __restrict__ slots, int sequences, int n_tokens) {
    tt_pdl_launch_dependents();
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    const int keep = taps - 1;
    float w[CONV_MAX_TAPS];
    float shift = 0.0f;
    if (c < channels) {                                          // filters are written by no kernel: fetched before the wait
#pragma unroll
        for (int j = 0; j < CONV_MAX_TAPS; ++j) w[j] = j < taps ? __ldg(weight + (size_t)c * taps + j) : 0.0f;
        shift = bias ? __ldg(bias + c) : 0.0f;
    }
    tt_pdl_wait();
    if (c >= channels) return;
    const int t0 = blockIdx.x * CONV_TILE, t1 = min(t0 + CONV_TILE, n_tokens);
    int b = tt_find_sequence(cu, sequences, t0);
    int first = cu[b], next = cu[b + 1];
    float win[CONV_MAX_TAPS];                                    // win[j], j < keep: the input (keep - j) tokens back
    auto fill = [&](int t) {                                     // the window as it stands before token t of sequence b
        const float* st = state + (size_t)slots[b] * slot_stride;
        const int i = t - first;
#pragma unroll
        for (int j = 0; j < CONV_MAX_TAPS; ++j) {
            if (j < keep) {
                const int s = i - keep + j;
                win[j] = s >= 0 ? rec_sum_slices(proj + (size_t)(first + s) * cols + col_off + c, splits, split_stride)
                                : st[(size_t)(keep + s) * channels + c];
            }
        }
    };
    fill(t0);
    for (int t = t0; t < t1; ++t) {
        if (t == next) {                                         // the next sequence starts here
            ++b;
            first = next;
            next = cu[b + 1];
            fill(t);
        }
        const float x = rec_sum_slices(proj + (size_t)t * cols + col_off + c, splits, split_stride);
        float acc = shift;
#pragma unroll
        for (int j = 0; j < CONV_MAX_TAPS; ++j)
            if (j <= keep) acc = fmaf(w[j], j < keep ? win[j] : x, acc);     // oldest input first, the token's own last
        out[(size_t)t * channels + c] = activation ? rec_silu(acc) : acc;
#pragma unroll
        for (int j = 0; j < CONV_MAX_TAPS - 1; ++j)
            if (j < keep) win[j] = j + 1 < keep ? win[j + 1] : x;
    }
}

// compute != 0: the sequence brings one token, whose output is computed here too
__global__ void causal_conv_state_kernel(const float* __restrict__ proj, int splits, size_t split_stride, int cols, int col_off,
                                         int channels, const float* __restrict__ weight, const float* __restrict__ bias, int taps,
                                         int activation, float* __restrict__ state, size_t slot_stride, float* __restrict__ out,
                                         const int* __restrict__ cu, const int* __restrict__ slots, int compute) {
    tt_pdl_launch_dependents();
    tt_pdl_wait();
    const int b = blockIdx.x;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int first = cu[b], n = cu[b + 1] - first;
    if (n <= 0) return;
    float* st = state + (size_t)slots[b] * slot_stride;
    const int keep = taps - 1;
    float next[CONV_MAX_TAPS];
    // the last `keep` entries of (old state, then this step's inputs)
#pragma unroll
    for (int e = 0; e < CONV_MAX_TAPS; ++e) {
        if (e < keep) {
            const int idx = n + e;              // index into the concatenation
            next[e] = idx < keep ? st[(size_t)idx * channels + c]
                                 : rec_sum_slices(proj + (size_t)(first + idx - keep) * cols + col_off + c, splits, split_stride);
        }
    }
    if (compute) {
        float acc = bias ? __ldg(bias + c) : 0.0f;
        for (int j = 0; j < keep; ++j) acc = fmaf(__ldg(weight + (size_t)c * taps + j), st[(size_t)j * channels + c], acc);
        const float x = rec_sum_slices(proj + (size_t)first * cols + col_off + c, splits, split_stride);
        acc = fmaf(__ldg(weight + (size_t)c * taps + keep), x, acc);
        out[(size_t)first * channels + c] = activation ? rec_silu(acc) : acc;
    }
#pragma unroll
    for (int e = 0; e < CONV_MAX_TAPS; ++e)
        if (e < keep) st[(size_t)e * channels + c] = next[e];
}

extern "C" int tt_causal_conv(const float* proj, int splits, long long split_stride, int cols, int col_off, int channels,
                              const float* weight, const float* bias, int taps, int activation, float* state,
                              long long slot_stride, float* out, const int* cu, const int* slots, int sequences, int n_tokens,
                              int one_token_each, cudaStream_t stream) {
    if (n_tokens <= 0 || channels <= 0) return 0;
    const int threads = 128;
    const unsigned bx = (unsigned)((channels + threads - 1) / threads);
    if (taps < 1 || taps > CONV_MAX_TAPS || bx > 65535) return (int)cudaErrorInvalidValue;
    if (!one_token_each) {
        tt_launch_pdl(causal_conv_kernel, dim3((n_tokens + CONV_TILE - 1) / CONV_TILE, bx), dim3(threads), 0, stream, proj, splits, (size_t)split_stride, cols, col_off,
                      channels, weight, bias, taps, activation, (const float*)state, (size_t)slot_stride, out, cu, slots, sequences, n_tokens);
    }
    if (taps > 1 || one_token_each)
        tt_launch_pdl(causal_conv_state_kernel, dim3(sequences, bx), dim3(threads), 0, stream, proj, splits, (size_t)split_stride, cols,
                      col_off, channels, weight, bias, taps, activation, state, (size_t)slot_stride, out, cu, slots, one_token_each);
    TT_LAUNCH_CHECK();
}

// ------------------------------------------------------------------------------------
// Mamba-2 recurrence.  Per head h (group g = h / (heads / groups)), state S [N x P], token t:
//   dt = softplus(dt_raw[t, h] + dt_bias[h])            (no clamp)
//   S  = exp(-exp(A_log[h]) * dt) * S + dt * B[t, g] x[t, h]^T
//   y[t, h] = S^T C[t, g] + D[h] * x[t, h]
// xbc: float32 [tokens][inner + 2 * groups * N] (x, then B, then C: the convolution's output);
// dt_raw: column dt_col of the projection's partial sums; state: [slots][heads][P][N].
// ------------------------------------------------------------------------------------
// G column groups of REC_LANES lanes per CTA, each owning C neighbouring columns: (32, 1) gives a sequence the most
// warps (one long prompt, decoding); (16, 4) reads a token's vectors from shared memory once for four columns, which is
// what bounds the kernel once the grid fills the GPU (batches of prompts).
// ROWS: every token brings a decay for each state row of its head (row_decay, float32 [tokens][groups * N], one more
// vector staged beside B and C) instead of one for the head; step sizes are one and there is no skip.
// BONUS (with ROWS): the token reads the state as it was before it and its own contribution by a weight for every state row of
// its head (row_bonus, float32 [groups * N]): y = (S + diag(bonus) B x^T)^T C, then S = diag(decay) S + B x^T.
template <int K, int G, int C, bool ROWS, bool BONUS>
__global__ void __launch_bounds__(G* REC_LANES)
mamba2_scan_kernel(const float* __restrict__ xbc, int xbc_cols, const float* __restrict__ proj, int splits, size_t split_stride,
                   int cols, int dt_col, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                   const float* __restrict__ d_skip, float* __restrict__ state, float* __restrict__ y,
                   const int* __restrict__ cu, const int* __restrict__ slots, int heads, int P, int N, int groups, int chunk,
                   int vec, const float* __restrict__ fixed_decay, const float* __restrict__ row_decay, const float* __restrict__ row_bonus) {
    tt_pdl_launch_dependents();
    tt_pdl_wait();
    extern __shared__ __align__(16) float rec_shared[];
    // two buffers of: B [chunk][NP], C [chunk][NP], (ROWS) decays [chunk][NP], x [chunk][TILE], decay [chunk], step [chunk];
    // rows are padded to NP = K * REC_LANES numbers and the padding is zero, so the token loop needs no bounds
    constexpr int NP = K * REC_LANES, TILE = G * C, VECTORS = ROWS ? 3 : 2;
    const int buffer_floats = VECTORS * chunk * NP + chunk * TILE + 2 * chunk;
    const int h = blockIdx.x, b = blockIdx.y, p0 = blockIdx.z * TILE;
    const int first = cu[b], n = cu[b + 1] - first;
    if (n <= 0) return;
    const int g = h / (heads / groups);
    const int inner = heads * P;
    const int lane = threadIdx.x % REC_LANES, col = (threadIdx.x / REC_LANES) * C;     // first of this group's columns in the tile
    const int width = min(TILE, P - p0);                        // columns of this tile that exist
    // fixed_decay: the head's decay is a constant and every step size is one (S = decay * S + B x^T, y = S^T C)
    const bool plain = ROWS || fixed_decay;                      // no step sizes, no skip
    const float fixed = fixed_decay ? __ldg(fixed_decay + h) : 0.0f;
    const float neg_a = plain ? 0.0f : -expf(__ldg(a_log + h)), bias = plain ? 0.0f : __ldg(dt_bias + h);
    const float skip = plain ? 0.0f : __ldg(d_skip + h);
    const bool vec_x = vec && (width & 3) == 0;
    float uv[BONUS ? K : 1];
    if constexpr (BONUS) {
#pragma unroll
        for (int i = 0; i < K; ++i) uv[i] = rec_row(lane, i) < N ? __ldg(row_bonus + (size_t)g * N + rec_row(lane, i)) : 0.0f;
    }

    auto stage = [&](int c0, float* base) {                      // asynchronous: B, C and x of tokens c0 .. of this sequence
        const int count = min(chunk, n - c0);
        const float* row = xbc + (size_t)(first + c0) * xbc_cols;
        rec_stage(base, NP, row + inner + g * N, xbc_cols, count, N, vec);
        rec_stage(base + chunk * NP, NP, row + inner + groups * N + g * N, xbc_cols, count, N, vec);
        if (ROWS) rec_stage(base + 2 * chunk * NP, NP, row_decay + ((size_t)(first + c0) * groups + g) * N, (size_t)groups * N, count, N, vec);
        rec_stage(base + VECTORS * chunk * NP, TILE, row + h * P + p0, xbc_cols, count, width, vec_x);
        rec_commit();
    };
    auto raw_step = [&](int c0) {                                // this thread's token of the chunk: the raw step size
        if (plain) return 0.0f;
        return rec_sum_slices(proj + (size_t)(first + c0 + threadIdx.x) * cols + dt_col + h, splits, split_stride);
    };
    auto put_scalars = [&](float* base, float raw) {
        if (ROWS) return;
        const float dt = fixed_decay ? 1.0f : rec_softplus(raw + bias);
        base[2 * chunk * NP + chunk * TILE + threadIdx.x] = fixed_decay ? fixed : expf(neg_a * dt);
        base[2 * chunk * NP + chunk * TILE + chunk + threadIdx.x] = dt;
    };

    for (int e = threadIdx.x; e < 2 * buffer_floats; e += blockDim.x) rec_shared[e] = 0.0f;
    __syncthreads();
    stage(0, rec_shared);
    float* S = state + (((size_t)slots[b] * heads + h) * P + p0 + col) * N;          // column c of the group lies c * N further
    float s[C][K];
#pragma unroll
    for (int c = 0; c < C; ++c) rec_load_column<K>(s[c], S + (size_t)(p0 + col + c < P ? c : 0) * N, lane, N, p0 + col + c < P);
    if (threadIdx.x < min(chunk, n)) put_scalars(rec_shared, raw_step(0));
    int it = 0;
    for (int c0 = 0; c0 < n; c0 += chunk, ++it) {
        float* cur = rec_shared + (it & 1) * buffer_floats;
        float* nxt = rec_shared + ((it + 1) & 1) * buffer_floats;
        const int count = min(chunk, n - c0);
        const int count_next = min(chunk, n - c0 - chunk);       // <= 0: this is the last chunk
        float raw_next = 0.0f;
        if (count_next > 0) {
            stage(c0 + chunk, nxt);                              // lands while this chunk is worked on
            if (threadIdx.x < count_next) raw_next = raw_step(c0 + chunk);
            rec_wait<1>();
        } else {
            rec_wait<0>();
        }
        __syncthreads();
        const float* Bs = cur;
        const float* Cs = cur + chunk * NP;
        const float* xs = cur + VECTORS * chunk * NP;
        const float* decay = xs + chunk * TILE;
        const float* step = decay + chunk;
        for (int k = 0; k < count; ++k) {
            const float a = ROWS ? 1.0f : decay[k], dt = ROWS ? 1.0f : step[k];
            float bv[K], cv[K], av[ROWS ? K : 1];                // all of the token's loads are asked for before the arithmetic
            rec_load_vector<K>(bv, Bs + k * NP, lane);
            rec_load_vector<K>(cv, Cs + k * NP, lane);
            if constexpr (ROWS) rec_load_vector<K>(av, Cs + (chunk + k) * NP, lane);
            float x[C], part[C];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                x[c] = p0 + col + c < P ? xs[k * TILE + col + c] : 0.0f;
                const float dx = dt * x[c];
                float part0 = 0.0f, part1 = 0.0f;                // two chains, so that neighbouring rows do not wait for each other
#pragma unroll
                for (int i = 0; i < K; i += 2) {
                    if constexpr (BONUS) {
                        const float b0 = dx * bv[i], b1 = dx * bv[i + 1];
                        part0 = fmaf(fmaf(uv[i], b0, s[c][i]), cv[i], part0);
                        part1 = fmaf(fmaf(uv[i + 1], b1, s[c][i + 1]), cv[i + 1], part1);
                        s[c][i] = fmaf(av[i], s[c][i], b0);
                        s[c][i + 1] = fmaf(av[i + 1], s[c][i + 1], b1);
                        continue;
                    }
                    s[c][i] = fmaf(dx, bv[i], (ROWS ? av[ROWS ? i : 0] : a) * s[c][i]);
                    part0 = fmaf(s[c][i], cv[i], part0);
                    s[c][i + 1] = fmaf(dx, bv[i + 1], (ROWS ? av[ROWS ? i + 1 : 0] : a) * s[c][i + 1]);
                    part1 = fmaf(s[c][i + 1], cv[i + 1], part1);
                }
                part[c] = part0 + part1;
            }
#pragma unroll
            for (int o = REC_LANES / 2; o > 0; o >>= 1) {        // the columns' sums over the lane group, side by side
#pragma unroll
                for (int c = 0; c < C; ++c) part[c] += __shfl_xor_sync(0xffffffffu, part[c], o);
            }
            if (lane == 0) {
#pragma unroll
                for (int c = 0; c < C; ++c)
                    if (p0 + col + c < P) y[(size_t)(first + c0 + k) * inner + h * P + p0 + col + c] = fmaf(skip, x[c], part[c]);
            }
        }
        if (count_next > 0 && threadIdx.x < count_next) put_scalars(nxt, raw_next);
        __syncthreads();                                         // this buffer may be filled again; the next one's scalars are written
    }
#pragma unroll
    for (int c = 0; c < C; ++c)
        if (p0 + col + c < P) rec_store_column<K>(s[c], S + (size_t)c * N, lane, N);
}

// Tokens staged at a time: 16 where two buffers of them (2 or 3 vectors of a state's rows, a column tile) fit the default 48 KB of shared memory, else 8 or 4.
static int rec_padded(int rows) { return rows <= 8 * REC_LANES ? 8 * REC_LANES : rows <= 16 * REC_LANES ? 16 * REC_LANES : 32 * REC_LANES; }
static size_t rec_shared_bytes(int rows, int chunk, int tile, int vectors) { return (size_t)2 * (vectors * chunk * rec_padded(rows) + chunk * tile + 2 * chunk) * sizeof(float); }
static int rec_chunk(int rows, int tile, int vectors) {
    int chunk = rows <= 128 ? REC_CHUNK : REC_CHUNK / 2;
    while (rec_shared_bytes(rows, chunk, tile, vectors) > 48 * 1024) chunk /= 2;
    return chunk;
}

constexpr int REC_WIDE_GROUPS = 16, REC_WIDE_COLS = 4;      // the form for grids that fill the GPU: 16 lane groups of 4 columns each

// Whether the grid of the (32, 1) form would fill the GPU more than twice over, so that the (16, 4) form pays
// (mode 0; 1 and 2 force the one or the other, for tests).  The wide form holds four columns of up to 128 rows.
static bool rec_wide(int mode, long long ctas, int rows) {
    if (rows > 16 * REC_LANES) return false;
    if (mode) return mode == 2;
    static int sms = 0;
    if (!sms) {
        int device = 0;
        cudaGetDevice(&device);
        if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device) != cudaSuccess || sms <= 0) sms = 148;
    }
    return ctas >= 2LL * sms;
}
static bool rec_aligned(const void* p, int a, int b, int c, int d) { return (((uintptr_t)p & 15) == 0) && !((a | b | c | d) & 3); }

static int mamba2_scan_launch(const float* xbc, int xbc_cols, const float* proj, int splits, long long split_stride, int cols,
                              int dt_col, const float* dt_bias, const float* a_log, const float* d_skip, float* state, float* y,
                              const int* cu, const int* slots, int sequences, int heads, int P, int N, int groups, int mode,
                              const float* fixed_decay, const float* row_decay, const float* row_bonus, cudaStream_t stream) {
    if (sequences <= 0) return 0;
    if (row_bonus && !row_decay) return (int)cudaErrorInvalidValue;
    if (N <= 0 || N > REC_MAX_ROWS || P <= 0 || groups <= 0 || heads % groups || sequences > 65535) return (int)cudaErrorInvalidValue;
    const int vec = rec_aligned(xbc, xbc_cols, N, P, 0) && ((uintptr_t)row_decay & 15) == 0 ? 1 : 0;          // every row piece starts on 16 bytes
    const bool wide = rec_wide(mode, (long long)heads * sequences * ((P + REC_COLS - 1) / REC_COLS), N);
    const int tile = wide ? REC_WIDE_GROUPS * REC_WIDE_COLS : REC_COLS;
    const dim3 grid(heads, sequences, (P + tile - 1) / tile), block((wide ? REC_WIDE_GROUPS : REC_COLS) * REC_LANES);
    const int vectors = row_decay ? 3 : 2, chunk = rec_chunk(N, tile, vectors);
    const size_t shared = rec_shared_bytes(N, chunk, tile, vectors);
#define TT_SCAN_FORM(K, G, C, ROWS, BONUS) tt_launch_pdl(mamba2_scan_kernel<K, G, C, ROWS, BONUS>, grid, block, shared, stream, xbc, xbc_cols, proj, splits, (size_t)split_stride, cols, dt_col, dt_bias, a_log, d_skip, state, y, cu, slots, heads, P, N, groups, chunk, vec, fixed_decay, row_decay, row_bonus)
#define TT_SCAN(K, G, C) do { if (row_bonus) TT_SCAN_FORM(K, G, C, true, true); else if (row_decay) TT_SCAN_FORM(K, G, C, true, false); else TT_SCAN_FORM(K, G, C, false, false); } while (0)
    if (wide) {
        if (N <= 8 * REC_LANES) TT_SCAN(8, REC_WIDE_GROUPS, REC_WIDE_COLS);
        else TT_SCAN(16, REC_WIDE_GROUPS, REC_WIDE_COLS);
    } else {
        if (N <= 8 * REC_LANES) TT_SCAN(8, REC_COLS, 1);
        else if (N <= 16 * REC_LANES) TT_SCAN(16, REC_COLS, 1);
        else TT_SCAN(32, REC_COLS, 1);
    }
#undef TT_SCAN
#undef TT_SCAN_FORM
    TT_LAUNCH_CHECK();
}

extern "C" int tt_mamba2_scan(const float* xbc, int xbc_cols, const float* proj, int splits, long long split_stride, int cols,
                              int dt_col, const float* dt_bias, const float* a_log, const float* d_skip, float* state, float* y,
                              const int* cu, const int* slots, int sequences, int heads, int P, int N, int groups, int mode,
                              cudaStream_t stream) {
    return mamba2_scan_launch(xbc, xbc_cols, proj, splits, split_stride, cols, dt_col, dt_bias, a_log, d_skip, state, y, cu, slots,
                              sequences, heads, P, N, groups, mode, nullptr, nullptr, nullptr, stream);
}

// ------------------------------------------------------------------------------------
// Linear attention with a fixed decay per head: S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, S [D x V] per head.
// It is the recurrence above with a constant decay, step size one, B = k, C = q, x = v and no skip, a group per head;
// vkq: float32 [tokens][heads * V + 2 * heads * D] (v, then k, then q: what tt_linear_attention_prepare writes);
// state: [slots][heads][V][D].
// ------------------------------------------------------------------------------------
extern "C" int tt_decay_scan(const float* vkq, int vkq_cols, const float* decay, float* state, float* out, const int* cu,
                             const int* slots, int sequences, int heads, int V, int D, int mode, cudaStream_t stream) {
    if (!decay) return (int)cudaErrorInvalidValue;
    return mamba2_scan_launch(vkq, vkq_cols, nullptr, 0, 0, 0, 0, nullptr, nullptr, nullptr, state, out, cu, slots, sequences, heads, V, D,
                              heads, mode, decay, nullptr, nullptr, stream);
}

// The same with decays that a token brings: S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, a_t one number per head and
// key channel (row_decay: float32 [tokens][heads * D]).  With a bonus (float32 [heads * D]) the token reads the state before it:
// o_t = (S_(t-1) + diag(bonus) k_t v_t^T)^T q_t, the update as before.
extern "C" int tt_row_decay_scan(const float* vkq, int vkq_cols, const float* row_decay, const float* bonus, float* state, float* out, const int* cu,
                                 const int* slots, int sequences, int heads, int V, int D, int mode, cudaStream_t stream) {
    if (!row_decay) return (int)cudaErrorInvalidValue;
    return mamba2_scan_launch(vkq, vkq_cols, nullptr, 0, 0, 0, 0, nullptr, nullptr, nullptr, state, out, cu, slots, sequences, heads, V, D,
                              heads, mode, nullptr, row_decay, bonus, stream);
}

// q, k and v of a linear attention from the partial sums of its input projection (columns [q | k | v | ...], q and k
// heads x D, v heads x V), as the scan reads them: [v | k | q].  activation != 0: silu on all three.  rotary_dim > 0:
// the first rotary_dim numbers of each head of q and k are rotated by the token's position (number i pairs with
// i + rotary_dim / 2, angle = position * inv_freq[i], float32).  q and k are multiplied by q_scale and k_scale after the rotation.
__global__ void linear_attention_prepare_kernel(const float* __restrict__ proj, int splits, size_t split_stride, int cols, int heads,
                                                int D, int V, int activation, const float* __restrict__ inv_freq, int rotary_dim,
                                                float q_scale, float k_scale, float* __restrict__ vkq, const int* __restrict__ cu,
                                                const int* __restrict__ len_before, int sequences) {
    tt_pdl_launch_dependents();
    const int t = blockIdx.x;
    int pos = 0;
    if (rotary_dim > 0) {
        const int b = tt_find_sequence(cu, sequences, t);
        pos = len_before[b] + (t - cu[b]);
    }
    tt_pdl_wait();
    const int qk = heads * D, hv = heads * V;
    const float* row = proj + (size_t)t * cols;
    float* out = vkq + (size_t)t * (hv + 2 * qk);
    const int half = rotary_dim >> 1;
    for (int j = blockIdx.y * blockDim.x + threadIdx.x; j < 2 * qk + hv; j += gridDim.y * blockDim.x) {
        float x = rec_sum_slices(row + j, splits, split_stride);
        if (activation) x = rec_silu(x);
        if (j >= 2 * qk) {                                       // v
            out[j - 2 * qk] = x;
            continue;
        }
        const bool is_k = j >= qk;
        const int i = (is_k ? j - qk : j) % D;
        if (i < rotary_dim) {
            const int pair = i < half ? j + half : j - half;
            float other = rec_sum_slices(row + pair, splits, split_stride);
            if (activation) other = rec_silu(other);
            float sn, cs;
            sincosf((float)pos * __ldg(inv_freq + (i < half ? i : i - half)), &sn, &cs);
            x = i < half ? x * cs - other * sn : x * cs + other * sn;
        }
        if (is_k) out[hv + (j - qk)] = x * k_scale;
        else out[hv + qk + j] = x * q_scale;
    }
}

extern "C" int tt_linear_attention_prepare(const float* proj, int splits, long long split_stride, int cols, int heads, int D, int V,
                                           int activation, const float* inv_freq, int rotary_dim, float q_scale, float k_scale, float* vkq,
                                           const int* cu, const int* len_before, int sequences, int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rotary_dim < 0 || rotary_dim > D || (rotary_dim & 1) || 2 * heads * D + heads * V > cols) return (int)cudaErrorInvalidValue;
    const int total = 2 * heads * D + heads * V;
    const int want = n_tokens >= 1024 ? (total + 1023) / 1024 : (total + 255) / 256;                // few tokens: a token's columns over more blocks
    const int tiles = want < 32 ? want : 32;
    tt_launch_pdl(linear_attention_prepare_kernel, dim3(n_tokens, tiles), dim3(256), 0, stream, proj, splits, (size_t)split_stride, cols, heads, D,
                  V, activation, inv_freq, rotary_dim, q_scale, k_scale, vkq, cu, len_before, sequences);
    TT_LAUNCH_CHECK();
}

// ------------------------------------------------------------------------------------
// Gated delta rule.  Per head h (query/key head g = h / (heads / qk_heads)), state S [D x V], token t:
//   q = q / sqrt(sum(q^2) + 1e-6) * D^-1/2,   k = k / sqrt(sum(k^2) + 1e-6)       (per head)
//   beta = sigmoid(b_raw[t, h]),   decay = exp(-exp(A_log[h]) * softplus(a_raw[t, h] + dt_bias[h]))
//   S = decay * S;  u = beta * (v - S^T k);  S = S + k u^T;  o[t, h] = S^T q
// qkv: float32 [tokens][2 * qk_heads * D + heads * V] (q, k, v: the convolutions' output); b_raw and
// a_raw: columns b_col + h and a_col + h of the projection's partial sums; state: [slots][heads][V][D].
// ROWS: a token's decay is a number for every state row (row_decay, float32 [tokens][heads * D], made beforehand), and the
// state's rows are multiplied by it one by one.
// ------------------------------------------------------------------------------------
template <int K, int G, int C, bool ROWS>
__global__ void __launch_bounds__(G* REC_LANES)
delta_scan_kernel(const float* __restrict__ qkv, int qkv_cols, const float* __restrict__ proj, int splits, size_t split_stride,
                  int cols, int b_col, int a_col, const float* __restrict__ dt_bias, const float* __restrict__ a_log,
                  float* __restrict__ state, float* __restrict__ o, const int* __restrict__ cu, const int* __restrict__ slots,
                  int heads, int qk_heads, int D, int V, int chunk, int vec, const float* __restrict__ row_decay) {
    tt_pdl_launch_dependents();
    tt_pdl_wait();
    extern __shared__ __align__(16) float rec_shared[];
    // two buffers of: q [chunk][DP], k [chunk][DP], (ROWS) decays [chunk][DP], v [chunk][TILE], decay [chunk], beta [chunk]; rows
    // are padded to DP = K * REC_LANES numbers and the padding is zero.  G lane groups of C neighbouring columns each, as above.
    constexpr int DP = K * REC_LANES, TILE = G * C, VECTORS = ROWS ? 3 : 2;
    const int buffer_floats = VECTORS * chunk * DP + chunk * TILE + 2 * chunk;
    const int h = blockIdx.x, b = blockIdx.y, p0 = blockIdx.z * TILE;
    const int first = cu[b], n = cu[b + 1] - first;
    if (n <= 0) return;
    const int g = h / (heads / qk_heads);
    const int lane = threadIdx.x % REC_LANES, col = (threadIdx.x / REC_LANES) * C;
    const int warp = threadIdx.x >> 5, wlane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const int width = min(TILE, V - p0);
    const float neg_a = ROWS ? 0.0f : -expf(__ldg(a_log + h)), bias = ROWS ? 0.0f : __ldg(dt_bias + h), q_scale = rsqrtf((float)D);
    const int k_off = qk_heads * D, v_off = 2 * qk_heads * D;
    const bool vec_v = vec && (width & 3) == 0;

    auto stage = [&](int c0, float* base) {
        const int count = min(chunk, n - c0);
        const float* row = qkv + (size_t)(first + c0) * qkv_cols;
        rec_stage(base, DP, row + g * D, qkv_cols, count, D, vec);
        rec_stage(base + chunk * DP, DP, row + k_off + g * D, qkv_cols, count, D, vec);
        if (ROWS) rec_stage(base + 2 * chunk * DP, DP, row_decay + ((size_t)(first + c0) * heads + h) * D, (size_t)heads * D, count, D, vec);
        rec_stage(base + VECTORS * chunk * DP, TILE, row + v_off + h * V + p0, qkv_cols, count, width, vec_v);
        rec_commit();
    };
    auto raw_pair = [&](int c0) {                                // this thread's token of the chunk: raw write strength, raw decay input
        const float* row = proj + (size_t)(first + c0 + threadIdx.x) * cols;
        return make_float2(rec_sum_slices(row + b_col + h, splits, split_stride), ROWS ? 0.0f : rec_sum_slices(row + a_col + h, splits, split_stride));
    };
    auto put_scalars = [&](float* base, float2 raw) {
        if (!ROWS) base[2 * chunk * DP + chunk * TILE + threadIdx.x] = expf(neg_a * rec_softplus(raw.y + bias));
        base[VECTORS * chunk * DP + chunk * TILE + chunk + threadIdx.x] = 1.0f / (1.0f + expf(-raw.x));
    };

    for (int e = threadIdx.x; e < 2 * buffer_floats; e += blockDim.x) rec_shared[e] = 0.0f;
    __syncthreads();
    stage(0, rec_shared);
    float* S = state + (((size_t)slots[b] * heads + h) * V + p0 + col) * D;
    float s[C][K];
#pragma unroll
    for (int c = 0; c < C; ++c) rec_load_column<K>(s[c], S + (size_t)(p0 + col + c < V ? c : 0) * D, lane, D, p0 + col + c < V);
    if (threadIdx.x < min(chunk, n)) put_scalars(rec_shared, raw_pair(0));
    int it = 0;
    for (int c0 = 0; c0 < n; c0 += chunk, ++it) {
        float* cur = rec_shared + (it & 1) * buffer_floats;
        float* nxt = rec_shared + ((it + 1) & 1) * buffer_floats;
        const int count = min(chunk, n - c0);
        const int count_next = min(chunk, n - c0 - chunk);
        float2 raw_next = make_float2(0.0f, 0.0f);
        if (count_next > 0) {
            stage(c0 + chunk, nxt);
            if (threadIdx.x < count_next) raw_next = raw_pair(c0 + chunk);
            rec_wait<1>();
        } else {
            rec_wait<0>();
        }
        __syncthreads();
        float* qs = cur;
        float* ks = cur + chunk * DP;
        // a warp per (token, q or k): sum of squares, scale to unit length (q also by D^-1/2)
        for (int item = warp; item < 2 * count; item += warps) {
            float* vecp = (item & 1 ? ks : qs) + (item >> 1) * DP;
            float sumsq = 0.0f;
            for (int r = wlane; r < D; r += 32) sumsq = fmaf(vecp[r], vecp[r], sumsq);
            const float scale = rsqrtf(tt_warp_sum(sumsq) + 1e-6f) * (item & 1 ? 1.0f : q_scale);
            for (int r = wlane; r < D; r += 32) vecp[r] *= scale;
        }
        __syncthreads();
        const float* vs = cur + VECTORS * chunk * DP;
        const float* decay = vs + chunk * TILE;
        const float* beta = decay + chunk;
        for (int k = 0; k < count; ++k) {
            const float a = ROWS ? 1.0f : decay[k], write = beta[k];
            float kv[K], qv[K], av[ROWS ? K : 1];                // all of the token's loads are asked for before the arithmetic
            rec_load_vector<K>(kv, ks + k * DP, lane);
            rec_load_vector<K>(qv, qs + k * DP, lane);
            if constexpr (ROWS) rec_load_vector<K>(av, ks + (chunk + k) * DP, lane);
            float part[C];
#pragma unroll
            for (int c = 0; c < C; ++c) {
                float part0 = 0.0f, part1 = 0.0f;
#pragma unroll
                for (int i = 0; i < K; i += 2) {
                    s[c][i] *= ROWS ? av[ROWS ? i : 0] : a;
                    part0 = fmaf(s[c][i], kv[i], part0);
                    s[c][i + 1] *= ROWS ? av[ROWS ? i + 1 : 0] : a;
                    part1 = fmaf(s[c][i + 1], kv[i + 1], part1);
                }
                part[c] = part0 + part1;
            }
#pragma unroll
            for (int o2 = REC_LANES / 2; o2 > 0; o2 >>= 1) {
#pragma unroll
                for (int c = 0; c < C; ++c) part[c] += __shfl_xor_sync(0xffffffffu, part[c], o2);
            }
#pragma unroll
            for (int c = 0; c < C; ++c) {
                const float u = write * ((p0 + col + c < V ? vs[k * TILE + col + c] : 0.0f) - part[c]);
                float part0 = 0.0f, part1 = 0.0f;
#pragma unroll
                for (int i = 0; i < K; i += 2) {
                    s[c][i] = fmaf(kv[i], u, s[c][i]);
                    part0 = fmaf(s[c][i], qv[i], part0);
                    s[c][i + 1] = fmaf(kv[i + 1], u, s[c][i + 1]);
                    part1 = fmaf(s[c][i + 1], qv[i + 1], part1);
                }
                part[c] = part0 + part1;
            }
#pragma unroll
            for (int o2 = REC_LANES / 2; o2 > 0; o2 >>= 1) {
#pragma unroll
                for (int c = 0; c < C; ++c) part[c] += __shfl_xor_sync(0xffffffffu, part[c], o2);
            }
            if (lane == 0) {
#pragma unroll
                for (int c = 0; c < C; ++c)
                    if (p0 + col + c < V) o[(size_t)(first + c0 + k) * (heads * V) + h * V + p0 + col + c] = part[c];
            }
        }
        if (count_next > 0 && threadIdx.x < count_next) put_scalars(nxt, raw_next);
        __syncthreads();
    }
#pragma unroll
    for (int c = 0; c < C; ++c)
        if (p0 + col + c < V) rec_store_column<K>(s[c], S + (size_t)c * D, lane, D);
}

// row_decay: the decays of the ROWS form (a_col, dt_bias and a_log are then not read), or null
extern "C" int tt_delta_scan(const float* qkv, int qkv_cols, const float* proj, int splits, long long split_stride, int cols,
                             int b_col, int a_col, const float* dt_bias, const float* a_log, const float* row_decay, float* state, float* o,
                             const int* cu, const int* slots, int sequences, int heads, int qk_heads, int D, int V, int mode,
                             cudaStream_t stream) {
    if (sequences <= 0) return 0;
    if (D <= 0 || D > REC_MAX_ROWS || V <= 0 || qk_heads <= 0 || heads % qk_heads || sequences > 65535) return (int)cudaErrorInvalidValue;
    const int vec = rec_aligned(qkv, qkv_cols, D, V, 0) && ((uintptr_t)row_decay & 15) == 0 ? 1 : 0;
    const bool wide = rec_wide(mode, (long long)heads * sequences * ((V + REC_COLS - 1) / REC_COLS), D);
    const int tile = wide ? REC_WIDE_GROUPS * REC_WIDE_COLS : REC_COLS;
    const dim3 grid(heads, sequences, (V + tile - 1) / tile), block((wide ? REC_WIDE_GROUPS : REC_COLS) * REC_LANES);
    const int vectors = row_decay ? 3 : 2, chunk = rec_chunk(D, tile, vectors);
    const size_t shared = rec_shared_bytes(D, chunk, tile, vectors);
#define TT_SCAN_FORM(K, G, C, ROWS) tt_launch_pdl(delta_scan_kernel<K, G, C, ROWS>, grid, block, shared, stream, qkv, qkv_cols, proj, splits, (size_t)split_stride, cols, b_col, a_col, dt_bias, a_log, state, o, cu, slots, heads, qk_heads, D, V, chunk, vec, row_decay)
#define TT_SCAN(K, G, C) do { if (row_decay) TT_SCAN_FORM(K, G, C, true); else TT_SCAN_FORM(K, G, C, false); } while (0)
    if (wide) {
        if (D <= 8 * REC_LANES) TT_SCAN(8, REC_WIDE_GROUPS, REC_WIDE_COLS);
        else TT_SCAN(16, REC_WIDE_GROUPS, REC_WIDE_COLS);
    } else {
        if (D <= 8 * REC_LANES) TT_SCAN(8, REC_COLS, 1);
        else if (D <= 16 * REC_LANES) TT_SCAN(16, REC_COLS, 1);
        else TT_SCAN(32, REC_COLS, 1);
    }
#undef TT_SCAN
#undef TT_SCAN_FORM
    TT_LAUNCH_CHECK();
}

// ------------------------------------------------------------------------------------
// The two recurrences with a decay per state row, for prompts: four tokens at a time.
//
// Within a block of tokens 0 .. 3 with decays g_t (vectors over the state's rows), P_t = g_0 * .. * g_t elementwise and
// s_(j,t) = g_(j+1) * .. * g_t, everything that reads the state reads the state before the block, S:
//   delta rule:        u_t = beta_t (v_t - S^T (P_t k_t) - sum_(j<t) [k_t . (s_(j,t) k_j)] u_j)
//   linear attention:  u_t = v_t
//   both:              o_t = S^T (P_t q_t) + sum_(j<=t) [q_t . (s_(j,t) k_j)] u_j,   S <- P_3 S + sum_j (s_(j,3) k_j) u_j^T
// so the eight (four) row products of a column are independent of one another and summed over its lanes together, where
// token by token each waits for the one before.  Only products of decays enter, never a quotient, so nothing can overflow
// that does not overflow in the recurrence itself, and all of it is float32.  The scaled vectors and the products in square
// brackets are the same for every column: four warps of the CTA prepare them for the 16 tokens ahead while four others walk
// the state through the 16 tokens before.
//
// A column's D state rows lie in the registers of RB_LANES neighbouring lanes, each lane holding the same rows of RB_COLS
// neighbouring columns; a CTA takes RB_TILE columns of one (sequence, head).  Blocks that are not full are filled with
// tokens that change nothing (k = q = 0, decay 1, beta 0).
// ------------------------------------------------------------------------------------
constexpr int RB_BLOCK = 4;                 // tokens of a block
constexpr int RB_BLOCKS = 4;                // blocks prepared at a time, one by each preparing warp
constexpr int RB_CHUNK = RB_BLOCK * RB_BLOCKS;
constexpr int RB_LANES = 16, RB_COLS = 2;
constexpr int RB_SCAN_WARPS = 4;
constexpr int RB_TILE = RB_SCAN_WARPS * (32 / RB_LANES) * RB_COLS;      // 16 columns
constexpr int RB_THREADS = 32 * (RB_SCAN_WARPS + RB_BLOCKS);
constexpr int RB_SCALARS = 16 + 16 + 4 + RB_BLOCK * RB_TILE + 4;        // A [4][4], B [4][4], beta [4], v [4][RB_TILE], padding

struct RowScan {
    const float* q;             // float32 rows of row_stride numbers: query/key head g at + g * D, value head h at + h * V
    const float* k;
    const float* v;
    size_t row_stride;
    const float* decay;         // [tokens][heads * D]
    const float* proj;          // delta rule: column b_col + h of the partial sums is the raw write strength
    int splits, cols, b_col;
    size_t split_stride;
    float q_scale;
    const float* bonus;         // [heads * D]: a token reads the state before it and its own contribution times this (not with the delta rule)
    float* state;               // [slots][heads][V][D]
    float* out;                 // [tokens][heads * V]
    const int* cu;
    const int* slots;
    int heads, qk_heads, D, V, vec;
};

__device__ __forceinline__ float rb_pick(const float (&a)[4], int i) { return i < 2 ? (i ? a[1] : a[0]) : (i == 2 ? a[2] : a[3]); }

// v[i], i < N, summed over N neighbouring lanes: lane l of the N ends up with the sum of v[l] (N a power of two)
template <int N>
__device__ __forceinline__ float rb_scatter_sum(float (&v)[N], int lane) {
#pragma unroll
    for (int o = N / 2; o > 0; o >>= 1) {
        const bool hi = lane & o;
#pragma unroll
        for (int i = 0; i < o; ++i) {
            const float send = hi ? v[i] : v[i + o], keep = hi ? v[i + o] : v[i];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    }
    return v[0];
}

// two bits a value: the (t, j) of the pair products, first A's (1,0) (2,0) (2,1) (3,0) (3,1) (3,2), then B's (0,0) (1,0) (1,1) ... (3,3)
constexpr uint32_t RB_T = 1u | 2u << 2 | 2u << 4 | 3u << 6 | 3u << 8 | 3u << 10 | 0u << 12 | 1u << 14 | 1u << 16 | 2u << 18 | 2u << 20 | 2u << 22 | 3u << 24 | 3u << 26 | 3u << 28 | 3u << 30;
constexpr uint32_t RB_J = 0u | 0u << 2 | 1u << 4 | 0u << 6 | 1u << 8 | 2u << 10 | 0u << 12 | 0u << 14 | 1u << 16 | 0u << 18 | 1u << 20 | 2u << 22 | 0u << 24 | 1u << 26 | 2u << 28 | 3u << 30;

template <int K, bool DELTA, bool BONUS>
__global__ void __launch_bounds__(RB_THREADS)
row_decay_blocks_kernel(const RowScan a) {
    tt_pdl_launch_dependents();
    tt_pdl_wait();
    extern __shared__ __align__(16) float rec_shared[];
    constexpr int DP = K * RB_LANES, E = DP / 32;               // rows padded to DP numbers; E of them in a preparing lane
    constexpr int VECTORS = (DELTA ? 3 : 2) * RB_BLOCK + 1;     // (P_t k_t) [4], P_t q_t [4], s_(j,3) k_j [4], P_3
    constexpr int BLOCK_FLOATS = VECTORS * DP + RB_SCALARS, BUFFER = RB_BLOCKS * BLOCK_FLOATS;
    constexpr int Q_AT = DELTA ? RB_BLOCK * DP : 0, KH_AT = Q_AT + RB_BLOCK * DP, P_AT = KH_AT + RB_BLOCK * DP, S_AT = VECTORS * DP;
    const int h = blockIdx.x, b = blockIdx.y, p0 = blockIdx.z * RB_TILE;
    const int first = a.cu[b], n = a.cu[b + 1] - first;
    if (n <= 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int D = a.D, V = a.V;
    const int chunks = (n + RB_CHUNK - 1) / RB_CHUNK;
    for (int e = threadIdx.x; e < 2 * BUFFER; e += RB_THREADS) rec_shared[e] = 0.0f;
    __syncthreads();

    if (warp >= RB_SCAN_WARPS) {
        // ------------------------------------------------------------ a block of four tokens prepared by a warp
        const int mine = warp - RB_SCAN_WARPS, g = h / (a.heads / a.qk_heads);
        auto row_of = [&](int e) { return E == 8 ? 4 * lane + 128 * (e >> 2) + (e & 3) : E * lane + e; };
        float q[4][E], k[4][E], d[4][E], v[2], raw = 0.0f;
        float bonus[BONUS ? E : 1];
        if constexpr (BONUS) {
#pragma unroll
            for (int e = 0; e < E; ++e) bonus[e] = row_of(e) < D ? __ldg(a.bonus + (size_t)h * D + row_of(e)) : 0.0f;
        }
        const int v_token = lane >> 3, v_col = 2 * (lane & 7);
        auto load_row = [&](float (&x)[E], const float* row, float missing, bool live) {
            constexpr int W = E < 4 ? E : 4;                    // numbers of a load
#pragma unroll
            for (int j = 0; j < E; j += W) {
                const int r = row_of(j);
                if (live && a.vec && r < D) {
                    if constexpr (W == 4) {
                        const float4 y = __ldg(reinterpret_cast<const float4*>(row + r));
                        x[j] = y.x; x[j + 1] = y.y; x[j + 2] = y.z; x[j + 3] = y.w;
                    } else {
                        const float2 y = __ldg(reinterpret_cast<const float2*>(row + r));
                        x[j] = y.x; x[j + 1] = y.y;
                    }
                } else {
#pragma unroll
                    for (int e = 0; e < W; ++e) x[j + e] = live && r + e < D ? __ldg(row + r + e) : missing;
                }
            }
        };
        auto fetch = [&](int c0) {
            const int t0 = c0 + mine * RB_BLOCK;
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const bool live = t0 + t < n;
                const size_t row = (size_t)(first + (live ? t0 + t : 0));
                load_row(q[t], a.q + row * a.row_stride + (size_t)g * D, 0.0f, live);
                load_row(k[t], a.k + row * a.row_stride + (size_t)g * D, 0.0f, live);
                load_row(d[t], a.decay + (row * a.heads + h) * D, 1.0f, live);
            }
            const bool live = t0 + v_token < n;
            const float* vr = a.v + (size_t)(first + t0 + v_token) * a.row_stride + (size_t)h * V + p0 + v_col;
            v[0] = live && p0 + v_col < V ? __ldg(vr) : 0.0f;
            v[1] = live && p0 + v_col + 1 < V ? __ldg(vr + 1) : 0.0f;
            if (DELTA && lane < 4 && t0 + lane < n)
                raw = rec_sum_slices(a.proj + (size_t)(first + t0 + lane) * a.cols + a.b_col + h, a.splits, a.split_stride);
        };
        fetch(0);
        for (int it = 0; it <= chunks; ++it) {
            if (it < chunks) {
                const int t0 = it * RB_CHUNK + mine * RB_BLOCK;
                float* base = rec_shared + (it & 1) * BUFFER + mine * BLOCK_FLOATS;
                constexpr int PAIRS = DELTA ? 32 : 16, A_AT = 8, B_AT = DELTA ? 14 : 0;
                float sums[PAIRS];                              // delta rule: |q_t|^2 [4], |k_t|^2 [4], A's six, B's ten; else B's ten
#pragma unroll
                for (int i = 0; i < PAIRS; ++i) sums[i] = 0.0f;
                float kh[4][E];
#pragma unroll
                for (int e = 0; e < E; ++e) {
                    if (DELTA) {
#pragma unroll
                        for (int t = 0; t < 4; ++t) {
                            sums[t] = fmaf(q[t][e], q[t][e], sums[t]);
                            sums[4 + t] = fmaf(k[t][e], k[t][e], sums[4 + t]);
                        }
                    }
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        float w = k[j][e];
                        sums[B_AT + j * (j + 1) / 2 + j] = fmaf(q[j][e], BONUS ? bonus[BONUS ? e : 0] * w : w, sums[B_AT + j * (j + 1) / 2 + j]);
#pragma unroll
                        for (int t = j + 1; t < 4; ++t) {
                            if (BONUS) {                        // the query meets the state before its own token's decay
                                sums[B_AT + t * (t + 1) / 2 + j] = fmaf(q[t][e], w, sums[B_AT + t * (t + 1) / 2 + j]);
                                w *= d[t][e];
                                continue;
                            }
                            w *= d[t][e];
                            if (DELTA) sums[A_AT + t * (t - 1) / 2 + j] = fmaf(k[t][e], w, sums[A_AT + t * (t - 1) / 2 + j]);
                            sums[B_AT + t * (t + 1) / 2 + j] = fmaf(q[t][e], w, sums[B_AT + t * (t + 1) / 2 + j]);
                        }
                        kh[j][e] = w;
                    }
                }
                float total = rb_scatter_sum<PAIRS>(sums, lane);
                float nq[4], nk[4], beta[4];
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    if (DELTA) {
                        nq[t] = rsqrtf(__shfl_sync(0xffffffffu, total, t) + 1e-6f) * a.q_scale;
                        nk[t] = rsqrtf(__shfl_sync(0xffffffffu, total, 4 + t) + 1e-6f);
                        beta[t] = t0 + t < n ? 1.0f / (1.0f + expf(-__shfl_sync(0xffffffffu, raw, t))) : 0.0f;
                    } else {
                        nq[t] = a.q_scale;
                        nk[t] = beta[t] = 1.0f;
                    }
                }
                if (!DELTA) total += __shfl_xor_sync(0xffffffffu, total, 16);
                const int pair = DELTA ? lane - 8 : lane + 6;   // its place among the 16 pairs
                if (pair >= (DELTA ? 0 : 6) && pair < 16) {
                    const int t = (RB_T >> (2 * pair)) & 3, j = (RB_J >> (2 * pair)) & 3;
                    const float into = pair < 6 ? rb_pick(beta, t) * rb_pick(nk, t) : rb_pick(nq, t);
                    base[S_AT + (pair < 6 ? 0 : 16) + t * 4 + j] = total * into * rb_pick(nk, j);
                }
                if (DELTA && lane < 4) base[S_AT + 32 + lane] = rb_pick(beta, lane);
                *reinterpret_cast<float2*>(base + S_AT + 36 + v_token * RB_TILE + v_col) = make_float2(v[0] * rb_pick(beta, v_token), v[1] * rb_pick(beta, v_token));
                float p[E];
#pragma unroll
                for (int e = 0; e < E; ++e) p[e] = 1.0f;
                auto put = [&](float* to, const float (&x)[E]) {
                    constexpr int W = E < 4 ? E : 4;
#pragma unroll
                    for (int j = 0; j < E; j += W) {
                        if constexpr (W == 4) *reinterpret_cast<float4*>(to + row_of(j)) = make_float4(x[j], x[j + 1], x[j + 2], x[j + 3]);
                        else *reinterpret_cast<float2*>(to + row_of(j)) = make_float2(x[j], x[j + 1]);
                    }
                };
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    float x[E];
#pragma unroll
                    for (int e = 0; e < E; ++e) {
                        const float before = p[e];
                        p[e] *= d[t][e];
                        x[e] = q[t][e] * (BONUS ? before : p[e]) * nq[t];
                    }
                    put(base + Q_AT + t * DP, x);
                    if (DELTA) {
#pragma unroll
                        for (int e = 0; e < E; ++e) x[e] = k[t][e] * p[e] * nk[t];
                        put(base + t * DP, x);
                    }
#pragma unroll
                    for (int e = 0; e < E; ++e) x[e] = kh[t][e] * nk[t];
                    put(base + KH_AT + t * DP, x);
                }
                put(base + P_AT, p);
                if (it + 1 < chunks) fetch((it + 1) * RB_CHUNK);          // lands while the others walk
            }
            __syncthreads();
        }
        return;
    }

    // ---------------------------------------------------------------- the state, walked through the prepared blocks
    const int l = lane & (RB_LANES - 1);
    const int col = (warp * (32 / RB_LANES) + lane / RB_LANES) * RB_COLS;          // first of this lane group's columns in the tile
    float* S = a.state + (((size_t)a.slots[b] * a.heads + h) * V + p0 + col) * D;
    float s[RB_COLS][K];
    auto state_row = [&](int i) { return 4 * l + 4 * RB_LANES * (i >> 2) + (i & 3); };
#pragma unroll
    for (int c = 0; c < RB_COLS; ++c)
#pragma unroll
        for (int i = 0; i < K; i += 4) {
            const int r = state_row(i);
            const bool live = p0 + col + c < V;
            if (live && !(D & 3) && r < D) {
                const float4 y = *reinterpret_cast<const float4*>(S + (size_t)c * D + r);
                s[c][i] = y.x; s[c][i + 1] = y.y; s[c][i + 2] = y.z; s[c][i + 3] = y.w;
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) s[c][i + e] = live && r + e < D ? S[(size_t)c * D + r + e] : 0.0f;
            }
        }
    __syncthreads();                                            // the first chunk is prepared
    for (int it = 1; it <= chunks; ++it) {
        const float* buffer = rec_shared + ((it - 1) & 1) * BUFFER;
        const int left = n - (it - 1) * RB_CHUNK;
        for (int blk = 0; blk < RB_BLOCKS && blk * RB_BLOCK < left; ++blk) {
            const float* base = buffer + blk * BLOCK_FLOATS;
            constexpr int DOTS = DELTA ? 16 : 8;                // [keys, queries][column][token], or [column][token]
            float dots[DOTS];
#pragma unroll
            for (int i = 0; i < DOTS; ++i) dots[i] = 0.0f;
#pragma unroll
            for (int i = 0; i < K; i += 4) {
#pragma unroll
                for (int t = 0; t < 4; ++t) {
                    const float4 y = *reinterpret_cast<const float4*>(base + Q_AT + t * DP + state_row(i));
#pragma unroll
                    for (int c = 0; c < RB_COLS; ++c) {
                        float& o = dots[(DELTA ? 8 : 0) + c * 4 + t];
                        o = fmaf(s[c][i], y.x, o); o = fmaf(s[c][i + 1], y.y, o); o = fmaf(s[c][i + 2], y.z, o); o = fmaf(s[c][i + 3], y.w, o);
                    }
                    if (DELTA) {
                        const float4 z = *reinterpret_cast<const float4*>(base + t * DP + state_row(i));
#pragma unroll
                        for (int c = 0; c < RB_COLS; ++c) {
                            float& o = dots[c * 4 + t];
                            o = fmaf(s[c][i], z.x, o); o = fmaf(s[c][i + 1], z.y, o); o = fmaf(s[c][i + 2], z.z, o); o = fmaf(s[c][i + 3], z.w, o);
                        }
                    }
                }
            }
            float dot = rb_scatter_sum<DOTS>(dots, l);
            if (!DELTA) dot += __shfl_xor_sync(0xffffffffu, dot, 8);
            const float* scalars = base + S_AT;
            float u[RB_COLS][4];
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const float2 y = *reinterpret_cast<const float2*>(scalars + 36 + t * RB_TILE + col);
                u[0][t] = y.x; u[1][t] = y.y;
            }
            if (DELTA) {
                const float4 beta = *reinterpret_cast<const float4*>(scalars + 32);
                const float4 a1 = *reinterpret_cast<const float4*>(scalars + 4), a2 = *reinterpret_cast<const float4*>(scalars + 8), a3 = *reinterpret_cast<const float4*>(scalars + 12);
#pragma unroll
                for (int c = 0; c < RB_COLS; ++c) {
                    float r[4];
#pragma unroll
                    for (int t = 0; t < 4; ++t) r[t] = __shfl_sync(0xffffffffu, dot, c * 4 + t, RB_LANES);
                    u[c][0] = fmaf(-beta.x, r[0], u[c][0]);
                    u[c][1] = fmaf(-a1.x, u[c][0], fmaf(-beta.y, r[1], u[c][1]));
                    u[c][2] = fmaf(-a2.y, u[c][1], fmaf(-a2.x, u[c][0], fmaf(-beta.z, r[2], u[c][2])));
                    u[c][3] = fmaf(-a3.z, u[c][2], fmaf(-a3.y, u[c][1], fmaf(-a3.x, u[c][0], fmaf(-beta.w, r[3], u[c][3]))));
                }
            }
            {                                                   // the lane that holds a query's row product writes its token's output
                const int t = l & 3, c = (l >> 2) & 1, token = (it - 1) * RB_CHUNK + blk * RB_BLOCK + t;
                const float4 w = *reinterpret_cast<const float4*>(scalars + 16 + 4 * t);
                float o = dot;
                o = fmaf(w.x, c ? u[1][0] : u[0][0], o);
                o = fmaf(w.y, c ? u[1][1] : u[0][1], o);
                o = fmaf(w.z, c ? u[1][2] : u[0][2], o);
                o = fmaf(w.w, c ? u[1][3] : u[0][3], o);
                if ((l >= 8) == DELTA && token < n && p0 + col + c < V) a.out[(size_t)(first + token) * (a.heads * V) + (size_t)h * V + p0 + col + c] = o;
            }
#pragma unroll
            for (int i = 0; i < K; i += 4) {
                const float4 p = *reinterpret_cast<const float4*>(base + P_AT + state_row(i));
#pragma unroll
                for (int c = 0; c < RB_COLS; ++c) { s[c][i] *= p.x; s[c][i + 1] *= p.y; s[c][i + 2] *= p.z; s[c][i + 3] *= p.w; }
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float4 y = *reinterpret_cast<const float4*>(base + KH_AT + j * DP + state_row(i));
#pragma unroll
                    for (int c = 0; c < RB_COLS; ++c) {
                        s[c][i] = fmaf(y.x, u[c][j], s[c][i]);
                        s[c][i + 1] = fmaf(y.y, u[c][j], s[c][i + 1]);
                        s[c][i + 2] = fmaf(y.z, u[c][j], s[c][i + 2]);
                        s[c][i + 3] = fmaf(y.w, u[c][j], s[c][i + 3]);
                    }
                }
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int c = 0; c < RB_COLS; ++c)
#pragma unroll
        for (int i = 0; i < K; i += 4) {
            const int r = state_row(i);
            if (p0 + col + c >= V) continue;
            if (!(D & 3) && r < D) {
                *reinterpret_cast<float4*>(S + (size_t)c * D + r) = make_float4(s[c][i], s[c][i + 1], s[c][i + 2], s[c][i + 3]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (r + e < D) S[(size_t)c * D + r + e] = s[c][i + e];
            }
        }
}

template <int K, bool DELTA, bool BONUS>
static int row_decay_blocks_launch(const RowScan& scan, int sequences, cudaStream_t stream) {
    constexpr size_t shared = (size_t)2 * RB_BLOCKS * (((DELTA ? 3 : 2) * RB_BLOCK + 1) * K * RB_LANES + RB_SCALARS) * sizeof(float);
    static bool allowed = false;
    if (!allowed) {
        const cudaError_t code = cudaFuncSetAttribute(row_decay_blocks_kernel<K, DELTA, BONUS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared);
        if (code != cudaSuccess) return (int)code;
        allowed = true;
    }
    tt_launch_pdl(row_decay_blocks_kernel<K, DELTA, BONUS>, dim3(scan.heads, sequences, (scan.V + RB_TILE - 1) / RB_TILE), dim3(RB_THREADS), shared, stream, scan);
    TT_LAUNCH_CHECK();
}

// delta != 0: the delta rule (q and k are made unit vectors, q also times q_scale; beta from proj); else linear attention (q times q_scale)
extern "C" int tt_row_decay_blocks(const float* q, const float* k, const float* v, long long row_stride, const float* decay, int delta,
                                   const float* proj, int splits, long long split_stride, int cols, int b_col, float q_scale, const float* bonus, float* state,
                                   float* out, const int* cu, const int* slots, int sequences, int heads, int qk_heads, int D, int V,
                                   cudaStream_t stream) {
    if (sequences <= 0) return 0;
    if (!q || !k || !v || !decay || D <= 0 || D > REC_MAX_ROWS || V <= 0 || qk_heads <= 0 || heads % qk_heads || sequences > 65535) return (int)cudaErrorInvalidValue;
    if (delta && (!proj || bonus)) return (int)cudaErrorInvalidValue;
    const uintptr_t bases = (uintptr_t)q | (uintptr_t)k | (uintptr_t)decay;
    const RowScan scan{q, k, v, (size_t)row_stride, decay, proj, splits, cols, b_col, (size_t)split_stride, q_scale, bonus, state, out, cu, slots,
                       heads, qk_heads, D, V, (bases & 15) == 0 && !(D & 3) && !(row_stride & 3) ? 1 : 0};
#define TT_BLOCKS(K) (delta ? row_decay_blocks_launch<K, true, false>(scan, sequences, stream) : bonus ? row_decay_blocks_launch<K, false, true>(scan, sequences, stream) \
                                                                                               : row_decay_blocks_launch<K, false, false>(scan, sequences, stream))
    if (D <= 4 * RB_LANES) return TT_BLOCKS(4);
    if (D <= 8 * RB_LANES) return TT_BLOCKS(8);
    return TT_BLOCKS(16);
#undef TT_BLOCKS
}

// ------------------------------------------------------------------------------------
// Products of low rank: z[t, j] = sum_r W[j, r] * x[t, r] with x the columns x_col .. x_col + rank - 1 of a projection's
// partial sums, and what is made of z at once (kind):
//   0: z      1: exp(-exp(a_log[h]) * softplus(z + bias[j])), h = j / per_head      2: sigmoid(z + bias[j]) ^ inv_tau
//   3: exp(-exp(z + bias[j]))
// x may pass tanh first (tanh_x).
// Up to two such products of one projection in one launch (blockIdx.z).  All float32; W is stored [rank][n] (transposed, so
// that neighbouring threads read neighbouring numbers) in either element type.
// ------------------------------------------------------------------------------------
struct LowRankPart {
    int x_col, rank, n, kind, per_head, tanh_x;
    const void* w;
    const float* bias;
    const float* a_log;
    float inv_tau;
    float* out;                 // float32 [tokens][n]
};
struct LowRankParts { LowRankPart part[2]; };

__device__ __forceinline__ float low_rank_finish(const LowRankPart& p, float z, int j) {
    if (p.kind == 1) return expf(-expf(__ldg(p.a_log + j / p.per_head)) * rec_softplus(z + __ldg(p.bias + j)));
    if (p.kind == 2) return expf(-rec_softplus(-(z + __ldg(p.bias + j))) * p.inv_tau);
    if (p.kind == 3) return expf(-expf(z + __ldg(p.bias + j)));
    return z;
}

// Few tokens (decoding): a CTA takes LRF_TOKENS tokens and LRF_COLS columns, whose rank its eight warps share among
// themselves.  The weights, which no kernel writes, are on their way to registers before the wait for the projection.
constexpr int LRF_TOKENS = 8, LRF_COLS = 64, LRF_WARPS = 8, LRF_RANKS = 128, LRF_EACH = LRF_RANKS / LRF_WARPS, LRF_SLICES = 16;

template <typename TW>
__global__ void __launch_bounds__(32 * LRF_WARPS)
low_rank_few_kernel(const float* __restrict__ proj, int splits, size_t split_stride, int cols, const LowRankParts parts, int n_tokens) {
    __shared__ __align__(16) float xs[LRF_RANKS * LRF_TOKENS];
    __shared__ float sums[LRF_WARPS][LRF_TOKENS][LRF_COLS];
    tt_pdl_launch_dependents();
    const LowRankPart p = blockIdx.z ? parts.part[1] : parts.part[0];
    const int j0 = blockIdx.y * LRF_COLS;
    if (j0 >= p.n) return;
    const int t0 = blockIdx.x * LRF_TOKENS, count = min(LRF_TOKENS, n_tokens - t0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int ja = j0 + lane, jb = ja + 32;
    const TW* w = reinterpret_cast<const TW*>(p.w);
    TW wa[LRF_EACH], wb[LRF_EACH];
    auto weights = [&](int r0) {
#pragma unroll
        for (int i = 0; i < LRF_EACH; ++i) {
            const int r = r0 + warp + i * LRF_WARPS;
            const TW* at = w + (size_t)r * p.n;
            wa[i] = r < p.rank && ja < p.n ? at[ja] : tt_from_float<TW>(0.0f);
            wb[i] = r < p.rank && jb < p.n ? at[jb] : tt_from_float<TW>(0.0f);
        }
    };
    weights(0);
    float acc[LRF_TOKENS][2];
#pragma unroll
    for (int t = 0; t < LRF_TOKENS; ++t) acc[t][0] = acc[t][1] = 0.0f;
    tt_pdl_wait();
    for (int r0 = 0; r0 < p.rank; r0 += LRF_RANKS) {
        if (r0) { __syncthreads(); weights(r0); }
        const int ranks = min(LRF_RANKS, p.rank - r0);
#pragma unroll
        for (int i = 0; i < LRF_RANKS * LRF_TOKENS / (32 * LRF_WARPS); ++i) {       // neighbouring threads: neighbouring ranks of one token
            const int e = threadIdx.x + i * 32 * LRF_WARPS, t = e / LRF_RANKS, r = e % LRF_RANKS;
            float total = 0.0f;
            if (t < count && r < ranks) {
                const float* from = proj + (size_t)(t0 + t) * cols + p.x_col + r0 + r;
                for (int s0 = 0; s0 < splits; s0 += LRF_SLICES) {                  // the slices' loads in flight together, added in order
                    float v[LRF_SLICES];
#pragma unroll
                    for (int s = 0; s < LRF_SLICES; ++s) v[s] = s0 + s < splits ? __ldg(from + (size_t)(s0 + s) * split_stride) : 0.0f;
#pragma unroll
                    for (int s = 0; s < LRF_SLICES; ++s) total += v[s];
                }
            }
            xs[r * LRF_TOKENS + t] = p.tanh_x ? tanhf(total) : total;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < LRF_EACH; ++i) {
            const float4* x4 = reinterpret_cast<const float4*>(xs + (warp + i * LRF_WARPS) * LRF_TOKENS);
            const float a = tt_to_float(wa[i]), b = tt_to_float(wb[i]);
#pragma unroll
            for (int q = 0; q < LRF_TOKENS / 4; ++q) {
                const float4 x = x4[q];
                acc[4 * q][0] = fmaf(x.x, a, acc[4 * q][0]);         acc[4 * q][1] = fmaf(x.x, b, acc[4 * q][1]);
                acc[4 * q + 1][0] = fmaf(x.y, a, acc[4 * q + 1][0]); acc[4 * q + 1][1] = fmaf(x.y, b, acc[4 * q + 1][1]);
                acc[4 * q + 2][0] = fmaf(x.z, a, acc[4 * q + 2][0]); acc[4 * q + 2][1] = fmaf(x.z, b, acc[4 * q + 2][1]);
                acc[4 * q + 3][0] = fmaf(x.w, a, acc[4 * q + 3][0]); acc[4 * q + 3][1] = fmaf(x.w, b, acc[4 * q + 3][1]);
            }
        }
    }
#pragma unroll
    for (int t = 0; t < LRF_TOKENS; ++t) { sums[warp][t][lane] = acc[t][0]; sums[warp][t][lane + 32] = acc[t][1]; }
    __syncthreads();
    for (int e = threadIdx.x; e < count * LRF_COLS; e += 32 * LRF_WARPS) {
        const int t = e / LRF_COLS, c = e % LRF_COLS;
        if (j0 + c >= p.n) continue;
        float z = 0.0f;
#pragma unroll
        for (int g = 0; g < LRF_WARPS; ++g) z += sums[g][t][c];
        p.out[(size_t)(t0 + t) * p.n + j0 + c] = low_rank_finish(p, z, j0 + c);
    }
}

// Prompts: the products themselves are matrix products like any other (the caller's); here are their inputs, columns of a
// projection's partial sums in the activation dtype, and what is made of their results, in place.
template <typename TAct>
__global__ void low_rank_inputs_kernel(const float* __restrict__ proj, int splits, size_t split_stride, int cols, int col0, int width0, int tanh0,
                                       TAct* __restrict__ out0, int col1, int width1, int tanh1, TAct* __restrict__ out1) {
    tt_pdl_launch_dependents();
    tt_pdl_wait();
    const float* row = proj + (size_t)blockIdx.x * cols;
    for (int r = threadIdx.x; r < width0 + width1; r += blockDim.x) {
        const bool second = r >= width0;
        float x = rec_sum_slices(row + (second ? col1 + r - width0 : col0 + r), splits, split_stride);
        if (second ? tanh1 : tanh0) x = tanhf(x);
        if (second) out1[(size_t)blockIdx.x * width1 + r - width0] = tt_from_float<TAct>(x);
        else out0[(size_t)blockIdx.x * width0 + r] = tt_from_float<TAct>(x);
    }
}

extern "C" int tt_low_rank_inputs(const float* proj, int splits, long long split_stride, int cols, int col0, int width0, int tanh0, void* out0,
                                  int col1, int width1, int tanh1, void* out1, int out_dtype, int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (width0 < 1 || width1 < 0 || col0 < 0 || col0 + width0 > cols || (width1 && (!out1 || col1 < 0 || col1 + width1 > cols))) return (int)cudaErrorInvalidValue;
    const int threads = width0 + width1 <= 64 ? 64 : (width0 + width1 <= 128 ? 128 : 256);
    if (out_dtype == TT_F32) tt_launch_pdl(low_rank_inputs_kernel<float>, dim3(n_tokens), dim3(threads), 0, stream, proj, splits, (size_t)split_stride, cols, col0, width0, tanh0, (float*)out0, col1, width1, tanh1, (float*)out1);
    else tt_launch_pdl(low_rank_inputs_kernel<__nv_bfloat16>, dim3(n_tokens), dim3(threads), 0, stream, proj, splits, (size_t)split_stride, cols, col0, width0, tanh0, (__nv_bfloat16*)out0, col1, width1, tanh1, (__nv_bfloat16*)out1);
    TT_LAUNCH_CHECK();
}

// out = finish(sum of z's slices), z float32 [splits][tokens][n]; out may be z's first slice
__global__ void low_rank_finish_kernel(const float* z, int splits, size_t split_stride, const LowRankPart p) {
    tt_pdl_launch_dependents();
    const int j = blockIdx.y * blockDim.x + threadIdx.x;
    if (j >= p.n) return;
    const float bias = __ldg(p.bias + j), rate = p.kind == 1 ? -expf(__ldg(p.a_log + j / p.per_head)) : 0.0f;
    tt_pdl_wait();
    const size_t at = (size_t)blockIdx.x * p.n + j;
    float x = bias;
    for (int s = 0; s < splits; ++s) x += z[(size_t)s * split_stride + at];
    p.out[at] = p.kind == 1 ? expf(rate * rec_softplus(x)) : p.kind == 2 ? expf(-rec_softplus(-x) * p.inv_tau) : expf(-expf(x));
}

extern "C" int tt_low_rank_finish(const float* z, int splits, long long split_stride, int n, int kind, int per_head, const float* bias,
                                  const float* a_log, float inv_tau, float* out, int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (n < 1 || kind < 1 || kind > 3 || !bias || (kind == 1 && (!a_log || per_head < 1))) return (int)cudaErrorInvalidValue;
    const LowRankPart p{0, 0, n, kind, per_head, 0, nullptr, bias, a_log, inv_tau, out};
    const int threads = 256;
    const unsigned blocks = (unsigned)((n + threads - 1) / threads);
    if (blocks > 65535) return (int)cudaErrorInvalidValue;
    tt_launch_pdl(low_rank_finish_kernel, dim3(n_tokens, blocks), dim3(threads), 0, stream, z, splits, (size_t)split_stride, p);
    TT_LAUNCH_CHECK();
}

extern "C" int tt_low_rank(const float* proj, int splits, long long split_stride, int cols, int n_parts, int w_dtype,
                           int x_col0, int rank0, int n0, int kind0, int per_head0, int tanh0, const void* w0, const float* bias0, const float* a_log0, float inv_tau0, float* out0,
                           int x_col1, int rank1, int n1, int kind1, int per_head1, int tanh1, const void* w1, const float* bias1, const float* a_log1, float inv_tau1, float* out1,
                           int n_tokens, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (n_parts < 1 || n_parts > 2) return (int)cudaErrorInvalidValue;
    LowRankParts parts;
    parts.part[0] = LowRankPart{x_col0, rank0, n0, kind0, per_head0, tanh0, w0, bias0, a_log0, inv_tau0, out0};
    parts.part[1] = n_parts > 1 ? LowRankPart{x_col1, rank1, n1, kind1, per_head1, tanh1, w1, bias1, a_log1, inv_tau1, out1} : parts.part[0];
    int widest = 0;
    for (int i = 0; i < n_parts; ++i) {
        const LowRankPart& p = parts.part[i];
        if (p.rank < 1 || p.n < 1 || p.x_col < 0 || p.x_col + p.rank > cols || p.kind < 0 || p.kind > 3) return (int)cudaErrorInvalidValue;
        if ((p.kind && !p.bias) || (p.kind == 1 && (!p.a_log || p.per_head < 1))) return (int)cudaErrorInvalidValue;
        widest = p.n > widest ? p.n : widest;
    }
    const dim3 grid((n_tokens + LRF_TOKENS - 1) / LRF_TOKENS, (widest + LRF_COLS - 1) / LRF_COLS, n_parts);
    if (grid.y > 65535) return (int)cudaErrorInvalidValue;
#define TT_LOW_RANK(T) tt_launch_pdl(low_rank_few_kernel<T>, grid, dim3(32 * LRF_WARPS), 0, stream, proj, splits, (size_t)split_stride, cols, parts, n_tokens)
    if (w_dtype == TT_F32) TT_LOW_RANK(float); else TT_LOW_RANK(__nv_bfloat16);
#undef TT_LOW_RANK
    TT_LAUNCH_CHECK();
}

// ------------------------------------------------------------------------------------
// Gate and group norm behind a recurrence.  y: float32 [tokens][width], cut into groups of `group`
// neighbouring columns; gate: columns gate_col .. gate_col + width - 1 of a projection's partial sums.
//   gate_first != 0:  v = y * silu(gate);  out = v / sqrt(mean_group(v^2) + eps) * w
//   gate_first == 0:  out = y / sqrt(mean_group(y^2) + eps) * w * silu(gate)
// w (float32 [weight_len]) is indexed by column modulo weight_len: one weight for the whole width, or one
// per position inside a head that all heads share.  One block per (token, group).
// ------------------------------------------------------------------------------------
template <typename TOut>
__global__ void gated_group_norm_kernel(const float* __restrict__ y, int width, int group, const float* __restrict__ proj,
                                        int splits, size_t split_stride, int cols, int gate_col,
                                        const float* __restrict__ weight, int weight_len, float eps, int gate_first,
                                        TOut* __restrict__ out, int gate_kind) {
    tt_pdl_launch_dependents();
    tt_pdl_wait();
    __shared__ float reduce[32];
    const int groups = width / group;
    const int t = blockIdx.x / groups, gi = blockIdx.x - t * groups;
    const float* yr = y + (size_t)t * width + (size_t)gi * group;
    const float* gr = proj + (size_t)t * cols + gate_col + (size_t)gi * group;
    float sumsq = 0.0f;
    for (int j = threadIdx.x; j < group; j += blockDim.x) {
        float v = yr[j];
        if (gate_first) v *= rec_gate(rec_sum_slices(gr + j, splits, split_stride), gate_kind);
        sumsq += v * v;
    }
    const float r = rsqrtf(tt_block_sum(sumsq, reduce) / (float)group + eps);
    TOut* o = out + (size_t)t * width + (size_t)gi * group;
    for (int j = threadIdx.x; j < group; j += blockDim.x) {
        const float gate = rec_gate(rec_sum_slices(gr + j, splits, split_stride), gate_kind);
        const float w = __ldg(weight + (gi * group + j) % weight_len);
        const float v = gate_first ? yr[j] * gate * r * w : yr[j] * r * w * gate;
        o[j] = tt_from_float<TOut>(v);
    }
}

// The same with a group's numbers kept in registers between the two passes (up to GN_VALUES per thread), so every
// input is loaded once and all loads of a thread are in flight together: the form for groups of up to 8,192 numbers.
constexpr int GN_VALUES = 8;

template <typename TOut>
__global__ void __launch_bounds__(1024)
gated_group_norm_reg_kernel(const float* __restrict__ y, int width, int group, const float* __restrict__ proj, int splits,
                            size_t split_stride, int cols, int gate_col, const float* __restrict__ weight, int weight_len,
                            float eps, int gate_first, TOut* __restrict__ out, int gate_kind) {
    tt_pdl_launch_dependents();
    tt_pdl_wait();
    __shared__ float reduce[32];
    const int groups = width / group;
    const int t = blockIdx.x / groups, gi = blockIdx.x - t * groups;
    const float* yr = y + (size_t)t * width + (size_t)gi * group;
    const float* gr = proj + (size_t)t * cols + gate_col + (size_t)gi * group;
    float v[GN_VALUES], gate[GN_VALUES];
    float sumsq = 0.0f;
#pragma unroll
    for (int e = 0; e < GN_VALUES; ++e) {
        const int j = threadIdx.x + e * blockDim.x;
        v[e] = 0.0f;
        gate[e] = 0.0f;
        if (j < group) {
            gate[e] = rec_gate(rec_sum_slices(gr + j, splits, split_stride), gate_kind);
            v[e] = gate_first ? yr[j] * gate[e] : yr[j];
            sumsq = fmaf(v[e], v[e], sumsq);
        }
    }
    const float r = rsqrtf(tt_block_sum(sumsq, reduce) / (float)group + eps);
    TOut* o = out + (size_t)t * width + (size_t)gi * group;
#pragma unroll
    for (int e = 0; e < GN_VALUES; ++e) {
        const int j = threadIdx.x + e * blockDim.x;
        if (j < group) {
            const float w = __ldg(weight + (gi * group + j) % weight_len);
            o[j] = tt_from_float<TOut>(gate_first ? v[e] * r * w : v[e] * r * w * gate[e]);
        }
    }
}

extern "C" int tt_gated_group_norm(const float* y, int n_tokens, int width, int group, const float* proj, int splits,
                                   long long split_stride, int cols, int gate_col, const float* weight, int weight_len, float eps,
                                   int gate_first, void* out, int out_dtype, int gate_kind, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (group <= 0 || width % group || weight_len <= 0) return (int)cudaErrorInvalidValue;
    const long long blocks = (long long)n_tokens * (width / group);
    if (blocks > 2147483647LL) return (int)cudaErrorInvalidValue;
    if (group <= 1024 * GN_VALUES) {
        int threads = (((group + 3) / 4 + 31) / 32) * 32;       // about four numbers a thread
        if (threads > 1024) threads = 1024;
        if (out_dtype == TT_F32)
            tt_launch_pdl(gated_group_norm_reg_kernel<float>, dim3((unsigned)blocks), dim3(threads), 0, stream, y, width, group, proj, splits, (size_t)split_stride, cols, gate_col, weight, weight_len, eps, gate_first, (float*)out, gate_kind);
        else
            tt_launch_pdl(gated_group_norm_reg_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(threads), 0, stream, y, width, group, proj, splits, (size_t)split_stride, cols, gate_col, weight, weight_len, eps, gate_first, (__nv_bfloat16*)out, gate_kind);
        TT_LAUNCH_CHECK();
    }
    const int threads = group >= 2048 ? 256 : (group >= 256 ? 128 : (group > 32 ? 64 : 32));
    if (out_dtype == TT_F32)
        tt_launch_pdl(gated_group_norm_kernel<float>, dim3((unsigned)blocks), dim3(threads), 0, stream, y, width, group, proj, splits, (size_t)split_stride, cols, gate_col, weight, weight_len, eps, gate_first, (float*)out, gate_kind);
    else
        tt_launch_pdl(gated_group_norm_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(threads), 0, stream, y, width, group, proj, splits, (size_t)split_stride, cols, gate_col, weight, weight_len, eps, gate_first, (__nv_bfloat16*)out, gate_kind);
    TT_LAUNCH_CHECK();
}

// ------------------------------------------------------------------------------------
// out[i] = wa * sum_s a[s][i] + wb * sum_s b[s][i]: two branches' outputs (each the partial sums of a
// product) weighted and added, float32.
// ------------------------------------------------------------------------------------
__global__ void weighted_pair_kernel(const float* __restrict__ a, int a_splits, size_t a_stride, float wa,
                                     const float* __restrict__ b, int b_splits, size_t b_stride, float wb,
                                     float* __restrict__ out, size_t total) {
    tt_pdl_launch_dependents();
    tt_pdl_wait();
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= total) return;
    out[i] = wa * rec_sum_slices(a + i, a_splits, a_stride) + wb * rec_sum_slices(b + i, b_splits, b_stride);
}

extern "C" int tt_weighted_pair(const float* a, int a_splits, long long a_stride, float wa, const float* b, int b_splits,
                                long long b_stride, float wb, float* out, long long total, cudaStream_t stream) {
    if (total <= 0) return 0;
    const int threads = 256;
    tt_launch_pdl(weighted_pair_kernel, dim3((unsigned)((total + threads - 1) / threads)), dim3(threads), 0, stream, a, a_splits,
                  (size_t)a_stride, wa, b, b_splits, (size_t)b_stride, wb, out, (size_t)total);
    TT_LAUNCH_CHECK();
}

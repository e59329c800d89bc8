// A residual stream in several copies ("hyper-connections"), with the RMS norm that reads it.
//
//   y    = scale * gain * sum_i delta[i][r]                       (a sublayer's output; gain: a factor per channel)
//   x'_t = sum_s mix[s][t] * x_s + write[t] * y                   (all copies at once from the old ones)
//   u    = sum_t read[t] * x'_t
//   out  = u * rsqrt(mean(u^2) + eps) * (weight + weight_offset)
// Copies: float32 [streams][tokens][hidden].  mix null: the copies stay (x'_t = x_t + write[t] * y); write and read null: ones.
// spread: only copy 0 is there so far and all copies start equal to it.  With `rows`, output row i comes from row rows[i] and no
// copy is written (the final norm at the wanted positions).  One block per output row; a thread only ever touches its own
// columns of the copies, so they are updated in place.  Everything is float32 until the one narrowing at the end.
#include "common.cuh"

constexpr int STREAMS_MAX = 16;         // largest count the general kernel takes
constexpr int STREAMS_FAST = 4;         // largest count with an instance of its own
constexpr int STREAM_THREADS = 512;

struct StreamPass {
    const float* delta;
    int splits;
    size_t split_stride;
    float scale;
    const float* gain;
    const float* mix;
    const float* write;
    const float* read;
    size_t stride;              // numbers between two copies
    int spread;
};

__device__ __forceinline__ void stream_store4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void stream_store4(__nv_bfloat16* p, const float4& v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 w;
    w.x = *reinterpret_cast<const uint32_t*>(&lo);
    w.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = w;
}
__device__ __forceinline__ void stream_fma(float4& a, float w, const float4& x) {
    a.x = fmaf(w, x.x, a.x); a.y = fmaf(w, x.y, a.y); a.z = fmaf(w, x.z, a.z); a.w = fmaf(w, x.w, a.w);
}

// S copies, PIECES float4 pieces of a row per thread, BATCH slices of the delta in flight together
template <typename TOut, int S, int PIECES, int BATCH>
__global__ void __launch_bounds__(STREAM_THREADS)
stream_norm_vec_kernel(float* __restrict__ streams, const StreamPass p, const float* __restrict__ weight, float weight_offset, float eps,
                       TOut* __restrict__ out, const int* __restrict__ rows, int hidden) {
    tt_pdl_launch_dependents();
    __shared__ float reduce[32];
    const int i = blockIdx.x, quads = hidden >> 2;
    // what no kernel writes is fetched while the previous kernel still runs
    float mix[S][S], write[S], read[S];
#pragma unroll
    for (int t = 0; t < S; ++t) {
        write[t] = p.scale * (p.write ? __ldg(p.write + t) : 1.0f);
        read[t] = p.read ? __ldg(p.read + t) : 1.0f;
#pragma unroll
        for (int s = 0; s < S; ++s) mix[s][t] = p.mix ? __ldg(p.mix + s * S + t) : (s == t ? 1.0f : 0.0f);
    }
    float4 w[PIECES], gain[PIECES];
#pragma unroll
    for (int v = 0; v < PIECES; ++v) {
        const int j = threadIdx.x + v * blockDim.x;
        gain[v] = make_float4(1.0f, 1.0f, 1.0f, 1.0f);
        if (j < quads) {
            w[v] = __ldg(reinterpret_cast<const float4*>(weight) + j);
            if (p.gain) gain[v] = __ldg(reinterpret_cast<const float4*>(p.gain) + j);
        }
    }
    tt_pdl_wait();
    const int r = rows ? rows[i] : i;
    const bool store = !rows && (p.splits > 0 || p.mix || p.spread);
    float4 u[PIECES];
    float sumsq = 0.0f;
#pragma unroll
    for (int v = 0; v < PIECES; ++v) {
        const int j = threadIdx.x + v * blockDim.x;
        if (j >= quads) continue;
        float4* at = reinterpret_cast<float4*>(streams + (size_t)r * hidden) + j;
        float4 x[S], y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (int s = 0; s < S; ++s) x[s] = at[p.spread ? 0 : (size_t)s * (p.stride >> 2)];
        const float4* d = reinterpret_cast<const float4*>(p.delta + (size_t)r * hidden) + j;
        for (int s0 = 0; s0 < p.splits; s0 += BATCH) {
            float4 q[BATCH];
#pragma unroll
            for (int e = 0; e < BATCH; ++e)
                if (s0 + e < p.splits) q[e] = __ldg(d + (size_t)(s0 + e) * (p.split_stride >> 2));
#pragma unroll
            for (int e = 0; e < BATCH; ++e)
                if (s0 + e < p.splits) { y.x += q[e].x; y.y += q[e].y; y.z += q[e].z; y.w += q[e].w; }
        }
        y.x *= gain[v].x; y.y *= gain[v].y; y.z *= gain[v].z; y.w *= gain[v].w;
        float4 sum = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
        for (int t = 0; t < S; ++t) {
            float4 n = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll
            for (int s = 0; s < S; ++s) stream_fma(n, mix[s][t], x[s]);
            stream_fma(n, write[t], y);
            if (store) at[(size_t)t * (p.stride >> 2)] = n;
            stream_fma(sum, read[t], n);
        }
        u[v] = sum;
        sumsq += sum.x * sum.x + sum.y * sum.y + sum.z * sum.z + sum.w * sum.w;
    }
    const float rstd = rsqrtf(tt_block_sum(sumsq, reduce) / (float)hidden + eps);
#pragma unroll
    for (int v = 0; v < PIECES; ++v) {
        const int j = threadIdx.x + v * blockDim.x;
        if (j >= quads) continue;
        const float o = weight_offset;
        stream_store4(out + (size_t)i * hidden + 4 * j, make_float4(u[v].x * rstd * (w[v].x + o), u[v].y * rstd * (w[v].y + o),
                                                                    u[v].z * rstd * (w[v].z + o), u[v].w * rstd * (w[v].w + o)));
    }
}

// any width and up to STREAMS_MAX copies; the row that the norm takes is kept in shared memory
template <typename TOut>
__global__ void __launch_bounds__(STREAM_THREADS)
stream_norm_kernel(float* __restrict__ streams, const StreamPass p, int copies, const float* __restrict__ weight, float weight_offset, float eps,
                   TOut* __restrict__ out, const int* __restrict__ rows, int hidden) {
    tt_pdl_launch_dependents();
    tt_pdl_wait();
    extern __shared__ float stream_row[];       // hidden, then 32 for the reduction
    const int i = blockIdx.x;
    const int r = rows ? rows[i] : i;
    const bool store = !rows && (p.splits > 0 || p.mix || p.spread);
    float sumsq = 0.0f;
    for (int j = threadIdx.x; j < hidden; j += blockDim.x) {
        float* at = streams + (size_t)r * hidden + j;
        float x[STREAMS_MAX], y = 0.0f, u = 0.0f;
#pragma unroll
        for (int s = 0; s < STREAMS_MAX; ++s) x[s] = s < copies ? at[p.spread ? 0 : (size_t)s * p.stride] : 0.0f;
        for (int s = 0; s < p.splits; ++s) y += p.delta[(size_t)s * p.split_stride + (size_t)r * hidden + j];
        if (p.gain) y *= p.gain[j];
#pragma unroll
        for (int t = 0; t < STREAMS_MAX; ++t) {
            if (t >= copies) continue;
            float n = 0.0f;
            if (p.mix) {
#pragma unroll
                for (int s = 0; s < STREAMS_MAX; ++s)
                    if (s < copies) n = fmaf(__ldg(p.mix + s * copies + t), x[s], n);
            } else {
                n = x[t];
            }
            n = fmaf(p.scale * (p.write ? __ldg(p.write + t) : 1.0f), y, n);
            if (store) at[(size_t)t * p.stride] = n;
            u = fmaf(p.read ? __ldg(p.read + t) : 1.0f, n, u);
        }
        stream_row[j] = u;
        sumsq += u * u;
    }
    const float rstd = rsqrtf(tt_block_sum(sumsq, stream_row + hidden) / (float)hidden + eps);
    for (int j = threadIdx.x; j < hidden; j += blockDim.x)
        out[(size_t)i * hidden + j] = tt_from_float<TOut>(stream_row[j] * rstd * (weight[j] + weight_offset));
}

extern "C" int tt_stream_norm(float* streams, int copies, long long stride, const float* delta, int splits, long long split_stride, float scale,
                              const float* gain, const float* mix, const float* write, const float* read, int spread, const float* weight,
                              float weight_offset, float eps, void* out, int out_dtype, const int* rows, int n_rows, int hidden,
                              cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (copies < 1 || copies > STREAMS_MAX || hidden <= 0 || !weight || !out) return (int)cudaErrorInvalidValue;
    const StreamPass p{delta, delta ? splits : 0, (size_t)split_stride, scale, gain, mix, write, read, (size_t)stride, spread};
    const uintptr_t bases = (uintptr_t)streams | (uintptr_t)delta | (uintptr_t)gain | (uintptr_t)weight | (uintptr_t)out;
    if (copies <= STREAMS_FAST && hidden % 4 == 0 && hidden <= 16 * STREAM_THREADS && stride % 4 == 0 && split_stride % 4 == 0 && (bases & 15) == 0) {
        int threads = ((hidden / 4 + 31) / 32) * 32;
        if (threads > STREAM_THREADS) threads = STREAM_THREADS;
        if (n_rows >= 1024) {                                     // prompts: smaller blocks of two pieces a thread (2,048 x 3,072, four copies: 78 us with
            const int fewest = (((hidden / 4 + 1) / 2 + 31) / 32) * 32;      // one piece, 50 with two, 72 with four; 8,192 x 2,048, two copies: 145, 76, 89)
            threads = fewest < 128 ? 128 : fewest > STREAM_THREADS ? STREAM_THREADS : fewest;
        }
        const int pieces = (hidden / 4 + threads - 1) / threads;
#define TT_STREAM(T, S, P, B) tt_launch_pdl(stream_norm_vec_kernel<T, S, P, B>, dim3(n_rows), dim3(threads), 0, stream, streams, p, weight, weight_offset, eps, (T*)out, rows, hidden)
#define TT_STREAMS(T, S) do { if (pieces == 1) TT_STREAM(T, S, 1, 8); else if (pieces == 2) TT_STREAM(T, S, 2, 2); else TT_STREAM(T, S, 4, 2); } while (0)
#define TT_STREAM_COUNT(T) do { switch (copies) { case 1: TT_STREAMS(T, 1); break; case 2: TT_STREAMS(T, 2); break; case 3: TT_STREAMS(T, 3); break; default: TT_STREAMS(T, 4); } } while (0)
        if (out_dtype == TT_F32) TT_STREAM_COUNT(float); else TT_STREAM_COUNT(__nv_bfloat16);
#undef TT_STREAM_COUNT
#undef TT_STREAMS
#undef TT_STREAM
        TT_LAUNCH_CHECK();
    }
    const size_t shared = ((size_t)hidden + 32) * sizeof(float);
    if (shared > 200 * 1024) return (int)cudaErrorInvalidValue;
    const int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
#define TT_STREAM_ANY(T)                                                                                                                    \
    do {                                                                                                                                    \
        if (shared > 48 * 1024) {                                                                                                           \
            const cudaError_t code = cudaFuncSetAttribute(stream_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)shared); \
            if (code != cudaSuccess) return (int)code;                                                                                      \
        }                                                                                                                                   \
        tt_launch_pdl(stream_norm_kernel<T>, dim3(n_rows), dim3(threads), shared, stream, streams, p, copies, weight, weight_offset, eps, (T*)out, rows, hidden); \
    } while (0)
    if (out_dtype == TT_F32) TT_STREAM_ANY(float); else TT_STREAM_ANY(__nv_bfloat16);
#undef TT_STREAM_ANY
    TT_LAUNCH_CHECK();
}

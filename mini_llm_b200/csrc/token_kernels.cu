// Kernels that read a token's identity beyond its embedding row, and the pass that puts a normed result onto the stream:
//   pair_embed      out[t] = scale * table[id_t] + pairs[row], row = (previous id * mul_prev + id * mul_cur) mod buckets, or
//                   the row `buckets` for a sequence's first token; the id before an entry's first token of the step is
//                   the request's state
//   token_gate      g[t, j] = gelu(W[j] . x[t]) * side[id_t, first + j]: a narrow product of the 32-bit stream, opened by
//                   a slice of the token's own row (steps of few tokens)
//   token_gate_rows the same behind a product that ran already: g[t, j] = gelu(z[t, j]) * side[id_t, first + j]
//   add_normed_norm hidden[t] += y[t] / rms(y[t]) * gain, and the norm of the row as it then is (another gain) as the
//                   next sublayer's input, in one pass
// Sums, norms and the stream are 32-bit; tables, matrices and results have the activations' type (float: the true 32-bit
// path; bfloat16: the serving path).  Every kernel is launched as a programmatic dependent of the kernel before it.
#include "common.cuh"

MLLM_DEFINE_ERROR_API(mllm_token)

// four consecutive entries of a row as 32-bit floats (the row starts on a boundary of four)
__device__ __forceinline__ float4 four(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 four(const bf16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void put_four(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put_four(bf16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 packed;
    packed.x = *reinterpret_cast<const unsigned*>(&a), packed.y = *reinterpret_cast<const unsigned*>(&b);
    *reinterpret_cast<uint2*>(p) = packed;
}

// ---------------------------------------------------------------------------
// A block per token.  Only the block of an entry's first token touches the request's state: it reads the id before the
// entry, then leaves the entry's last id there.
// ---------------------------------------------------------------------------
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
pair_embed_kernel(float* __restrict__ out, const int* __restrict__ ids, const int* __restrict__ positions,
                  const int* __restrict__ token_item, const int* __restrict__ item_slot, const int* __restrict__ item_offset,
                  const int* __restrict__ item_count, const T* __restrict__ table, const T* __restrict__ pairs,
                  int* __restrict__ state, long long buckets, long long mul_prev, long long mul_cur, int width, float scale) {
    dependents_may_start();
    wait_for_earlier_kernels();
    const int t = blockIdx.x, id = ids[t], item = token_item[t], offset = item_offset[item];
    long long row = buckets;
    if (t > offset) {
        if (positions[t] > 0) row = ((long long)ids[t - 1] * mul_prev + (long long)id * mul_cur) % buckets;
    } else {
        const int slot = item_slot[item];
        const int before = state[slot];
        if (positions[t] > 0) row = ((long long)before * mul_prev + (long long)id * mul_cur) % buckets;
        __syncthreads();                                     // every thread has read the state
        if (threadIdx.x == 0) state[slot] = ids[offset + item_count[item] - 1];
    }
    const T* a = table + (long)id * width;
    const T* b = pairs + (long)row * width;
    float* o = out + (long)t * width;
    if (VEC) {
        for (int c = threadIdx.x * 4; c < width; c += blockDim.x * 4) {
            const float4 u = four(a + c), v = four(b + c);
            put_four(o + c, make_float4(fmaf(u.x, scale, v.x), fmaf(u.y, scale, v.y), fmaf(u.z, scale, v.z), fmaf(u.w, scale, v.w)));
        }
    } else {
        for (int c = threadIdx.x; c < width; c += blockDim.x) o[c] = fmaf(to_f32(a[c]), scale, to_f32(b[c]));
    }
}

extern "C" int mllm_token_pair_embed(float* out, const int* ids, const int* positions, const int* token_item, const int* item_slot,
                                     const int* item_offset, const int* item_count, const void* table, const void* pairs, int* state,
                                     long buckets, long mul_prev, long mul_cur, int n_tokens, int width, float scale, int dtype,
                                     void* stream) {
    if (n_tokens <= 0) return 0;
    if (width <= 0 || buckets <= 0 || mul_prev < 0 || mul_cur < 0) return fail("pair_embed: the sizes must be positive, the factors not negative");
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = width % 4 == 0 && (((unsigned long long)out | (unsigned long long)table | (unsigned long long)pairs) & 15ull) == 0;
    const int threads = width >= 1024 ? 256 : 64;
#define RUN(T, VEC)                                                                                                              \
    launch_kernel(g_dependent_launch != 0, pair_embed_kernel<T, VEC>, dim3(n_tokens), dim3(threads), 0, s, out, ids, positions,   \
                  token_item, item_slot, item_offset, item_count, (const T*)table, (const T*)pairs, state, (long long)buckets,    \
                  (long long)mul_prev, (long long)mul_cur, width, scale)
    if (dtype == DT_F32) { if (vec) RUN(float, true); else RUN(float, false); }
    else if (dtype == DT_BF16) { if (vec) RUN(bf16, true); else RUN(bf16, false); }
    else return fail("pair_embed: unknown dtype");
#undef RUN
    return check_launch("pair_embed_kernel");
}

// ---------------------------------------------------------------------------
// A warp takes one row of the gate matrix and TOKENS tokens: the row is read once for all of them, the tokens' rows
// come from shared memory.
// ---------------------------------------------------------------------------
constexpr int GATE_WARPS = 8;

template <typename T, int TOKENS, bool VEC>
__global__ void __launch_bounds__(GATE_WARPS * 32)
token_gate_kernel(T* __restrict__ out, const float* __restrict__ x, const T* __restrict__ w, const T* __restrict__ side, long ld_side,
                  const int* __restrict__ ids, int first, int dim, int width, int n_tokens) {
    dependents_may_start();
    wait_for_earlier_kernels();
    extern __shared__ __align__(16) float rows[];            // [TOKENS][width]
    const int t0 = blockIdx.y * TOKENS, n_here = min(TOKENS, n_tokens - t0);
    for (int i = threadIdx.x; i < n_here * width; i += blockDim.x) rows[i] = x[(long)t0 * width + i];
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int j = blockIdx.x * GATE_WARPS + warp;
    if (j >= dim) return;
    float z[TOKENS];
#pragma unroll
    for (int g = 0; g < TOKENS; g++) z[g] = 0.0f;
    const T* row = w + (long)j * width;
    if (VEC) {
#pragma unroll 4
        for (int c = lane * 4; c < width; c += 128) {
            const float4 a = four(row + c);
#pragma unroll
            for (int g = 0; g < TOKENS; g++) {
                if (g >= n_here) continue;
                const float4 b = four(rows + g * width + c);
                z[g] = fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, z[g]))));
            }
        }
    } else {
        for (int c = lane; c < width; c += 32)
#pragma unroll
            for (int g = 0; g < TOKENS; g++)
                if (g < n_here) z[g] = fmaf(to_f32(row[c]), rows[g * width + c], z[g]);
    }
#pragma unroll
    for (int g = 0; g < TOKENS; g++) {
        if (g >= n_here) continue;
        const float sum = warp_sum(z[g]);
        if (lane == 0) out[(long)(t0 + g) * dim + j] = from_f32<T>(gelu_tanh_f(sum) * to_f32(side[(long)ids[t0 + g] * ld_side + first + j]));
    }
}

extern "C" int mllm_token_gate(void* out, const float* x, const void* w, const void* side, long ld_side, const int* ids, int first,
                               int dim, int width, int n_tokens, int dtype, void* stream) {
    if (n_tokens <= 0) return 0;
    if (dim <= 0 || width <= 0 || first < 0) return fail("token_gate: sizes must be positive");
    const int tokens = n_tokens <= 8 ? 1 : 4;
    int group = tokens;
    if (sizeof(float) * (size_t)width * group > 48 * 1024) group = 1;
    const size_t shared = sizeof(float) * (size_t)width * group;
    if (shared > 48 * 1024) return fail("token_gate: the token does not fit shared memory");
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid((dim + GATE_WARPS - 1) / GATE_WARPS, (n_tokens + group - 1) / group);
    if (grid.y > 65535) return fail("token_gate: too many tokens for one launch");
    const bool vec = width % 4 == 0 && ((unsigned long long)w & 15ull) == 0;
#define RUN(T, G, VEC)                                                                                                           \
    launch_kernel(g_dependent_launch != 0, token_gate_kernel<T, G, VEC>, grid, dim3(GATE_WARPS * 32), shared, s, (T*)out, x,      \
                  (const T*)w, (const T*)side, ld_side, ids, first, dim, width, n_tokens)
#define PICK(T)                                                                                                                  \
    do {                                                                                                                         \
        if (group == 4) { if (vec) RUN(T, 4, true); else RUN(T, 4, false); }                                                     \
        else { if (vec) RUN(T, 1, true); else RUN(T, 1, false); }                                                                \
    } while (0)
    if (dtype == DT_F32) PICK(float);
    else if (dtype == DT_BF16) PICK(bf16);
    else return fail("token_gate: unknown dtype");
#undef PICK
#undef RUN
    return check_launch("token_gate_kernel");
}

template <typename T, int N>
__global__ void __launch_bounds__(256)
token_gate_rows_kernel(T* __restrict__ out, const float* __restrict__ z, const T* __restrict__ side, long ld_side,
                       const int* __restrict__ ids, int first, int dim, long n) {
    dependents_may_start();
    wait_for_earlier_kernels();
    const long i = ((long)blockIdx.x * blockDim.x + threadIdx.x) * N;
    if (i >= n) return;
    const long t = i / dim;
    const T* e = side + (long)ids[t] * ld_side + first + i % dim;
    if (N == 4) {
        const float4 a = four(z + i), b = four(e);
        put_four(out + i, make_float4(gelu_tanh_f(a.x) * b.x, gelu_tanh_f(a.y) * b.y, gelu_tanh_f(a.z) * b.z, gelu_tanh_f(a.w) * b.w));
    } else {
        out[i] = from_f32<T>(gelu_tanh_f(z[i]) * to_f32(*e));
    }
}

extern "C" int mllm_token_gate_rows(void* out, const float* z, const void* side, long ld_side, const int* ids, int first, int dim,
                                    int n_tokens, int dtype, void* stream) {
    if (n_tokens <= 0) return 0;
    if (dim <= 0 || first < 0) return fail("token_gate_rows: sizes must be positive");
    const long n = (long)n_tokens * dim;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = dim % 4 == 0 && ld_side % 4 == 0 && first % 4 == 0 &&
                     (((unsigned long long)out | (unsigned long long)z | (unsigned long long)side) & 15ull) == 0;
    const int per = vec ? 4 : 1;
#define RUN(T, N)                                                                                                                \
    launch_kernel(g_dependent_launch != 0, token_gate_rows_kernel<T, N>, dim3((unsigned)((n / N + 255) / 256)), dim3(256), 0, s,  \
                  (T*)out, z, (const T*)side, ld_side, ids, first, dim, n)
    if (dtype == DT_F32) { if (per == 4) RUN(float, 4); else RUN(float, 1); }
    else if (dtype == DT_BF16) { if (per == 4) RUN(bf16, 4); else RUN(bf16, 1); }
    else return fail("token_gate_rows: unknown dtype");
#undef RUN
    return check_launch("token_gate_rows_kernel");
}

// ---------------------------------------------------------------------------
// A block per row; the row of the new stream lies in shared memory between its sum and its norm.
// ---------------------------------------------------------------------------
template <typename T, bool VEC>
__global__ void __launch_bounds__(512)
add_normed_norm_kernel(float* __restrict__ hidden, const float* __restrict__ y, const float* __restrict__ gain, float eps,
                       T* __restrict__ normed, const float* __restrict__ next_gain, float next_eps, int width) {
    dependents_may_start();
    wait_for_earlier_kernels();
    __shared__ float scratch[33];
    extern __shared__ __align__(16) float row[];             // [width]
    const long at = (long)blockIdx.x * width;
    float sq = 0.0f;
    if (VEC) {
        for (int c = threadIdx.x * 4; c < width; c += blockDim.x * 4) {
            const float4 v = four(y + at + c);
            put_four(row + c, v);
            sq = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, sq))));
        }
    } else {
        for (int c = threadIdx.x; c < width; c += blockDim.x) {
            const float v = y[at + c];
            row[c] = v;
            sq = fmaf(v, v, sq);
        }
    }
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)width + eps);
    float next = 0.0f;
    if (VEC) {
        for (int c = threadIdx.x * 4; c < width; c += blockDim.x * 4) {      // (a thread's own entries of the row)
            const float4 v = four(row + c), g = four(gain + c);
            float4 h = four(hidden + at + c);
            h.x = fmaf(v.x * inv, g.x, h.x), h.y = fmaf(v.y * inv, g.y, h.y), h.z = fmaf(v.z * inv, g.z, h.z), h.w = fmaf(v.w * inv, g.w, h.w);
            put_four(hidden + at + c, h);
            put_four(row + c, h);
            next = fmaf(h.x, h.x, fmaf(h.y, h.y, fmaf(h.z, h.z, fmaf(h.w, h.w, next))));
        }
    } else {
        for (int c = threadIdx.x; c < width; c += blockDim.x) {
            const float h = fmaf(row[c] * inv, gain[c], hidden[at + c]);
            hidden[at + c] = h;
            row[c] = h;
            next = fmaf(h, h, next);
        }
    }
    if (normed == nullptr) return;
    const float next_inv = 1.0f / sqrtf(block_sum(next, scratch) / (float)width + next_eps);
    if (VEC) {
        for (int c = threadIdx.x * 4; c < width; c += blockDim.x * 4) {
            const float4 h = four(row + c), g = four(next_gain + c);
            put_four(normed + at + c, make_float4(h.x * next_inv * g.x, h.y * next_inv * g.y, h.z * next_inv * g.z, h.w * next_inv * g.w));
        }
    } else {
        for (int c = threadIdx.x; c < width; c += blockDim.x) normed[at + c] = from_f32<T>(row[c] * next_inv * next_gain[c]);
    }
}

extern "C" int mllm_token_add_normed_norm_takes(int width) { return width > 0 && sizeof(float) * (size_t)width <= 47 * 1024; }

extern "C" int mllm_token_add_normed_norm(float* hidden, const float* y, const float* gain, float eps, void* normed,
                                          const float* next_gain, float next_eps, int width, int n_rows, int dtype, void* stream) {
    if (n_rows <= 0) return 0;
    if (!mllm_token_add_normed_norm_takes(width)) return fail("add_normed_norm: the row does not fit shared memory");
    if (normed != nullptr && next_gain == nullptr) return fail("add_normed_norm: a norm needs its gain");
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = width % 4 == 0 && (((unsigned long long)hidden | (unsigned long long)y | (unsigned long long)gain |
                                         (unsigned long long)normed | (unsigned long long)next_gain) & 15ull) == 0;
    const int threads = width >= 2048 ? 512 : (width >= 512 ? 256 : 128);
    const size_t shared = sizeof(float) * (size_t)width;
#define RUN(T, VEC)                                                                                                              \
    launch_kernel(g_dependent_launch != 0, add_normed_norm_kernel<T, VEC>, dim3(n_rows), dim3(threads), shared, s, hidden, y,     \
                  gain, eps, (T*)normed, next_gain, next_eps, width)
    if (dtype == DT_F32) { if (vec) RUN(float, true); else RUN(float, false); }
    else if (dtype == DT_BF16) { if (vec) RUN(bf16, true); else RUN(bf16, false); }
    else return fail("add_normed_norm: unknown dtype");
#undef RUN
    return check_launch("add_normed_norm_kernel");
}

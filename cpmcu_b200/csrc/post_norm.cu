// The residual stream of layers whose norm comes after the sum, and the embedding that starts it.
//
//   post_norm     x <- rms_norm(alpha * x + scale * a) * w       (a sublayer's output a, scaled channel by channel)
//   embed_norm    x  = rms_norm(table[token] * s + bigram[row(previous token, token)]) * w
//
// Both leave x in fp32 (the stream) and a copy in the storage type, which is what the next sublayer's products read:
// with the norm after the sum a sublayer reads the stream itself.  Sums and norms are fp32.
#include "common.cuh"

// Norms the row in ``row_cache`` (hidden floats, ss: this thread's part of the sum of squares; w null: no weight) into x
// and y (either may be null).
template <typename T>
__device__ __forceinline__ void norm_row_out(const float* row_cache, float ss, float* scratch, const float* __restrict__ w,
                                             float* __restrict__ x, T* __restrict__ y, int hidden, float eps, bool norm) {
    const float r = norm ? 1.0f / sqrtf(block_sum(ss, scratch) / (float)hidden + eps) : 1.f;
    if ((hidden & 3) == 0) {
        for (int c = 4 * threadIdx.x; c < hidden; c += 4 * blockDim.x) {      // what this thread itself wrote into row_cache
            float4 v = *reinterpret_cast<const float4*>(row_cache + c);
            if (norm) {
                const float4 g = load4(w + c);
                v = make_float4(v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w);
            }
            store4(x + c, v);
            if (y) store4(y + c, v);
        }
    } else {
        for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
            const float v = norm ? row_cache[c] * r * w[c] : row_cache[c];
            x[c] = v;
            if (y) y[c] = from_f32<T>(v);
        }
    }
}

template <typename T>
__global__ void post_norm_kernel(float* __restrict__ x, const T* __restrict__ a, float alpha, const float* __restrict__ scale,
                                 const float* __restrict__ w, T* __restrict__ y, int hidden, float eps) {
    extern __shared__ float row_cache[];   // hidden floats + 33
    pdl_launch_dependents();
    pdl_wait();
    float* xr = x + (int64_t)blockIdx.x * hidden;
    const T* ar = a + (int64_t)blockIdx.x * hidden;
    float ss = 0.f;
    if ((hidden & 3) == 0) {
        for (int c = 4 * threadIdx.x; c < hidden; c += 4 * blockDim.x) {
            const float4 v = load4(xr + c);
            float4 d = load4(ar + c);
            if (scale) {
                const float4 g = load4(scale + c);
                d = make_float4(d.x * g.x, d.y * g.y, d.z * g.z, d.w * g.w);
            }
            d = make_float4(fmaf(alpha, v.x, d.x), fmaf(alpha, v.y, d.y), fmaf(alpha, v.z, d.z), fmaf(alpha, v.w, d.w));
            *reinterpret_cast<float4*>(row_cache + c) = d;
            ss = fmaf(d.x, d.x, fmaf(d.y, d.y, fmaf(d.z, d.z, fmaf(d.w, d.w, ss))));
        }
    } else {
        for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
            const float v = fmaf(alpha, xr[c], to_f32(ar[c]) * (scale ? scale[c] : 1.f));
            row_cache[c] = v;
            ss = fmaf(v, v, ss);
        }
    }
    norm_row_out<T>(row_cache, ss, row_cache + hidden, w, xr, y ? y + (int64_t)blockIdx.x * hidden : nullptr, hidden, eps, true);
}

template <typename T>
static int launch_post_norm(float* x, const void* a, float alpha, const float* scale, const float* w, void* y, int n_tokens, int hidden,
                            float eps, cudaStream_t stream) {
    const size_t smem = (size_t)(hidden + 36) * sizeof(float);
    if (smem > 227 * 1024) return CPM_BAD_ARGUMENT;
    auto kern = post_norm_kernel<T>;
    static bool configured[kMaxDevices] = {};
    if (smem > 48 * 1024)
        if (int e = ensure_dynamic_smem(kern, 227 * 1024, configured)) return e;
    const int threads = hidden >= 4096 ? 512 : (hidden >= 1024 ? 256 : 128);
    cpm_launch(kLaunchNorm, kern, n_tokens, threads, smem, stream, x, (const T*)a, alpha, scale, w, (T*)y, hidden, eps);
    return launch_status();
}

// x fp32 [tokens, hidden] in place; a [tokens, hidden] in the storage type; scale fp32 [hidden] or null; w fp32 [hidden];
// y [tokens, hidden] in the storage type or null.
CPM_API int cpm_post_norm(float* x, const void* a, float alpha, const float* scale, const float* w, void* y, int n_tokens, int hidden,
                          float eps, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return CPM_OK;
    if (hidden < 1) return CPM_BAD_ARGUMENT;
    if (dtype == CPM_BF16) return launch_post_norm<bf16>(x, a, alpha, scale, w, y, n_tokens, hidden, eps, stream);
    return launch_post_norm<float>(x, a, alpha, scale, w, y, n_tokens, hidden, eps, stream);
}

// ---------------------------------------------------------------------------
// The embedding's row of a token plus a row of a second table that a hash of (the token before, the token) picks:
// (previous * mul_prev + token * mul_cur) mod buckets, or row ``buckets`` for a sequence's first token.  The token before a
// step's first one comes from prev_state [slots]; the block of a sequence's first token of the step reads it and then
// leaves the sequence's last token there, so no other block touches it.
// ---------------------------------------------------------------------------
template <typename T>
__global__ void embed_norm_kernel(const int* __restrict__ ids, const T* __restrict__ table, float scale, const T* __restrict__ bigram,
                                  int64_t buckets, int64_t mul_prev, int64_t mul_cur, int* __restrict__ prev_state,
                                  const int* __restrict__ positions, const int* __restrict__ token_seq, const int* __restrict__ cu_q,
                                  const int* __restrict__ slots, const float* __restrict__ w, float* __restrict__ x, T* __restrict__ y,
                                  int hidden, float eps) {
    extern __shared__ float row_cache[];   // hidden floats + 33
    __shared__ int64_t bigram_row;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int id = ids[t];
    if (bigram != nullptr) {
        if (threadIdx.x == 0) {
            const int seq = token_seq[t], first = cu_q[seq], slot = slots[seq];
            int64_t row = buckets;
            if (positions[t] != 0) {
                const int64_t prev = t > first ? ids[t - 1] : prev_state[slot];
                row = (prev * mul_prev + (int64_t)id * mul_cur) % buckets;
                if (row < 0) row += buckets;
            }
            if (t == first) prev_state[slot] = ids[cu_q[seq + 1] - 1];
            bigram_row = row;
        }
        __syncthreads();
    }
    const T* src = table + (int64_t)id * hidden;
    const T* more = bigram != nullptr ? bigram + bigram_row * hidden : nullptr;
    float ss = 0.f;
    if ((hidden & 3) == 0) {
        for (int c = 4 * threadIdx.x; c < hidden; c += 4 * blockDim.x) {
            const float4 e = load4(src + c);
            float4 v = make_float4(e.x * scale, e.y * scale, e.z * scale, e.w * scale);
            if (more) {
                const float4 b = load4(more + c);
                v = make_float4(v.x + b.x, v.y + b.y, v.z + b.z, v.w + b.w);
            }
            *reinterpret_cast<float4*>(row_cache + c) = v;
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
    } else {
        for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
            const float v = to_f32(src[c]) * scale + (more ? to_f32(more[c]) : 0.f);
            row_cache[c] = v;
            ss = fmaf(v, v, ss);
        }
    }
    norm_row_out<T>(row_cache, ss, row_cache + hidden, w, x + (int64_t)t * hidden, y ? y + (int64_t)t * hidden : nullptr, hidden, eps,
                    w != nullptr);
}

template <typename T>
static int launch_embed_norm(const int* ids, const void* table, float scale, const void* bigram, int64_t buckets, int64_t mul_prev,
                             int64_t mul_cur, int* prev_state, const int* positions, const int* token_seq, const int* cu_q,
                             const int* slots, const float* w, float* x, void* y, int n_tokens, int hidden, float eps,
                             cudaStream_t stream) {
    const size_t smem = (size_t)(hidden + 36) * sizeof(float);
    if (smem > 227 * 1024) return CPM_BAD_ARGUMENT;
    auto kern = embed_norm_kernel<T>;
    static bool configured[kMaxDevices] = {};
    if (smem > 48 * 1024)
        if (int e = ensure_dynamic_smem(kern, 226 * 1024, configured)) return e;
    const int threads = hidden >= 4096 ? 512 : (hidden >= 1024 ? 256 : 128);
    cpm_launch(kLaunchOther, kern, n_tokens, threads, smem, stream, ids, (const T*)table, scale, (const T*)bigram, buckets, mul_prev,
               mul_cur, prev_state, positions, token_seq, cu_q, slots, w, x, (T*)y, hidden, eps);
    return launch_status();
}

// bigram [buckets + 1, hidden] with prev_state int32 [slots], or null; w fp32 [hidden] or null (no norm); x fp32, y in the
// storage type or null, both [tokens, hidden].
CPM_API int cpm_embed_norm(const int* ids, const void* table, float scale, const void* bigram, int64_t buckets, int64_t mul_prev,
                           int64_t mul_cur, int* prev_state, const int* positions, const int* token_seq, const int* cu_q,
                           const int* slots, const float* w, float* x, void* y, int n_tokens, int hidden, float eps, int dtype,
                           cudaStream_t stream) {
    if (n_tokens <= 0) return CPM_OK;
    if (hidden < 1 || (bigram != nullptr && (buckets < 1 || prev_state == nullptr))) return CPM_BAD_ARGUMENT;
    if (dtype == CPM_BF16)
        return launch_embed_norm<bf16>(ids, table, scale, bigram, buckets, mul_prev, mul_cur, prev_state, positions, token_seq, cu_q,
                                       slots, w, x, y, n_tokens, hidden, eps, stream);
    return launch_embed_norm<float>(ids, table, scale, bigram, buckets, mul_prev, mul_cur, prev_state, positions, token_seq, cu_q, slots,
                                    w, x, y, n_tokens, hidden, eps, stream);
}

// Linear attention with one fixed decay per head and no softmax (retention), and what stands around its recurrence.
//
//   S_t = a_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t         S [d, dv] per head, fp32, kept per sequence [slots, heads, d, dv]
//
// q and k are turned by the token's position first (pairs (i, i + rot/2) or, ``adjacent``, (2i, 2i + 1); cosine and sine times a
// magnitude) and k is scaled; each head's o is divided by its root mean square and multiplied by SiLU of a gate.
//
//   retention_step   one token per sequence (decode): rotation, state update, read-out, norm and gate in one kernel;
//                    a block holds one head of one token, its threads sweep the state once (read, update, write)
//   rotate_scale     the rotation and scaling alone, in place (for prompts)
//   retention tiles  prompts, by tiles of 64 consecutive tokens of a sequence, all of it fp32 FMA work:
//     tile_kv        what a tile adds to the state:  U = sum_j a^(n-1-j) k_j v_j^T        (n: the tile's tokens)
//     tile_scan      walks a sequence's tiles: leaves the state before each tile in U's place, S <- a^n S + U, and the last
//                    state in the sequence's slot
//     tile_out       o_i = a^(i+1) S^T q_i + sum_(j <= i) a^(i-j) (q_i . k_j) v_j, then norm and gate
// A tile's work depends on nothing but its own tokens and the state before it, so tiles run side by side; a portion of any
// size and a batch of any sequences give the same sums up to their order.
#include "common.cuh"

constexpr int kRetTile = 64;         // tokens of a tile (the step's query tiles)
constexpr int kRetPitch = 68;        // floats of a staged row of 64: 16-byte aligned, neighbouring rows in other banks

__device__ __forceinline__ float ret_silu(float v) { return v / (1.0f + expf(-v)); }

// ---------------------------------------------------------------------------
// In place on fp32 rows of ``stride`` floats: ``heads`` heads of d channels from the row's start on; the first ``rot`` channels
// of each are turned, and the heads from ``first_scaled`` on are multiplied by ``factor``.  One block a token.
// ---------------------------------------------------------------------------
__global__ void rotate_scale_kernel(float* __restrict__ x, int64_t stride, const int* __restrict__ positions, int heads, int d, int rot,
                                    const float* __restrict__ inv_freq, float magnitude, int adjacent, int first_scaled, float factor) {
    extern __shared__ float2 rs_cs[];
    pdl_launch_dependents();
    pdl_wait();
    const int half = rot >> 1;
    const int p = positions[blockIdx.x];
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, cn;
        sincosf((float)p * inv_freq[i], &sn, &cn);
        rs_cs[i] = make_float2(cn * magnitude, sn * magnitude);
    }
    __syncthreads();
    float* row = x + (int64_t)blockIdx.x * stride;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
    for (int h = warp; h < heads; h += n_warps) {
        float* hp = row + (int64_t)h * d;
        const float f = h >= first_scaled ? factor : 1.f;
        for (int i = lane; i < half; i += 32) {
            const int a = adjacent ? 2 * i : i, b = adjacent ? 2 * i + 1 : i + half;
            const float u = hp[a], v = hp[b];
            hp[a] = (u * rs_cs[i].x - v * rs_cs[i].y) * f;
            hp[b] = (v * rs_cs[i].x + u * rs_cs[i].y) * f;
        }
        if (f != 1.f)
            for (int c = rot + lane; c < d; c += 32) hp[c] *= f;
    }
}

CPM_API int cpm_rotate_scale(float* x, int64_t stride, const int* positions, int n_tokens, int heads, int d, int rot,
                             const float* inv_freq, float magnitude, int adjacent, int first_scaled, float factor, cudaStream_t stream) {
    if (n_tokens <= 0) return CPM_OK;
    if (heads < 1 || d < 1 || rot < 0 || (rot & 1) || rot > d || rot > 8192 || (rot && !inv_freq) || stride < (int64_t)heads * d)
        return CPM_BAD_ARGUMENT;
    cpm_launch(kLaunchRope, rotate_scale_kernel, dim3(n_tokens), dim3(256), (size_t)rot * sizeof(float) + 16, stream, x, stride, positions,
               heads, d, rot, inv_freq, magnitude, adjacent, first_scaled, factor);
    return launch_status();
}

// ---------------------------------------------------------------------------
// One token per sequence.  proj rows (fp32): q at 0, k at heads * d, v behind it, the gate behind v, as the layer's one
// product leaves them (not rotated).  A thread owns VEC neighbouring columns of the state and every RG-th of its rows.
// ---------------------------------------------------------------------------
constexpr int kStepThreads = 256;
constexpr int kStepFlight = 8;       // rows of the state a thread asks for before it uses the first

template <typename T, int VEC>
__global__ void __launch_bounds__(kStepThreads)
retention_step_kernel(const float* __restrict__ proj, int64_t stride, const float* __restrict__ decay, float* __restrict__ state,
                      const int* __restrict__ positions, const int* __restrict__ token_seq, const int* __restrict__ slots,
                      T* __restrict__ out, int heads, int d, int dv, int rot, const float* __restrict__ inv_freq, float magnitude,
                      int adjacent, float k_factor, float eps) {
    extern __shared__ float st_smem[];            // q [d], k [d], partial sums [RG][dv], read-out [dv], 33 for the block's sum
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    float* qs = st_smem;
    float* ks = qs + d;
    const int groups = dv / VEC, rows_at_once = kStepThreads / groups;
    float* part = ks + d;
    float* os = part + rows_at_once * dv;
    float* scratch = os + dv;
    const int p = positions[t];
    const float* row = proj + (int64_t)t * stride;
    const float* qr = row + (int64_t)h * d;
    const float* kr = qr + (int64_t)heads * d;
    const float* vr = row + 2 * (int64_t)heads * d + (int64_t)h * dv;
    const float* gr = vr + (int64_t)heads * dv;
    const int half = rot >> 1;
    for (int i = tid; i < half; i += kStepThreads) {
        float sn, cn;
        sincosf((float)p * inv_freq[i], &sn, &cn);
        sn *= magnitude;
        cn *= magnitude;
        const int a = adjacent ? 2 * i : i, b = adjacent ? 2 * i + 1 : i + half;
        const float qa = qr[a], qb = qr[b], ka = kr[a], kb = kr[b];
        qs[a] = qa * cn - qb * sn;
        qs[b] = qb * cn + qa * sn;
        ks[a] = (ka * cn - kb * sn) * k_factor;
        ks[b] = (kb * cn + ka * sn) * k_factor;
    }
    for (int c = rot + tid; c < d; c += kStepThreads) {
        qs[c] = qr[c];
        ks[c] = kr[c] * k_factor;
    }
    const int cg = tid % groups, rg = tid / groups;
    const bool live = rg < rows_at_once;
    float* st = state + ((int64_t)slots[token_seq[t]] * heads + h) * d * dv + (int64_t)cg * VEC;
    const bool fresh = p == 0;
    const float a1 = decay[h];
    float v[VEC], o[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
        v[j] = vr[cg * VEC + j];
        o[j] = 0.f;
    }
    __syncthreads();
    if (live) {
        for (int c0 = rg; c0 < d; c0 += kStepFlight * rows_at_once) {
            float s[kStepFlight][VEC];
#pragma unroll
            for (int u = 0; u < kStepFlight; ++u) {
                const int c = c0 + u * rows_at_once;
#pragma unroll
                for (int j = 0; j < VEC; ++j) s[u][j] = 0.f;
                if (c < d && !fresh) {
                    if (VEC == 4) {
                        const float4 f = load4(st + (int64_t)c * dv);
                        s[u][0] = f.x; s[u][1 % VEC] = f.y; s[u][2 % VEC] = f.z; s[u][3 % VEC] = f.w;
                    } else s[u][0] = st[(int64_t)c * dv];
                }
            }
#pragma unroll
            for (int u = 0; u < kStepFlight; ++u) {
                const int c = c0 + u * rows_at_once;
                if (c < d) {
                    const float kc = ks[c], qc = qs[c];
#pragma unroll
                    for (int j = 0; j < VEC; ++j) {
                        s[u][j] = fmaf(a1, s[u][j], kc * v[j]);
                        o[j] = fmaf(qc, s[u][j], o[j]);
                    }
                    if (VEC == 4) store4(st + (int64_t)c * dv, make_float4(s[u][0], s[u][1 % VEC], s[u][2 % VEC], s[u][3 % VEC]));
                    else st[(int64_t)c * dv] = s[u][0];
                }
            }
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) part[rg * dv + cg * VEC + j] = o[j];
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = tid; c < dv; c += kStepThreads) {
        float sum = 0.f;
        for (int r = 0; r < rows_at_once; ++r) sum += part[r * dv + c];
        os[c] = sum;
        ss = fmaf(sum, sum, ss);
    }
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)dv + eps);
    T* dst = out + ((int64_t)t * heads + h) * dv;
    for (int c = tid; c < dv; c += kStepThreads) dst[c] = from_f32<T>(os[c] * f * ret_silu(gr[c]));
}

// Whether the one-kernel step takes heads of d key and dv value channels.
CPM_API int cpm_retention_step_sizes(int d, int dv) {
    const int groups = dv % 4 == 0 ? dv / 4 : dv;
    return d >= 1 && d <= 1024 && dv >= 1 && groups <= kStepThreads ? 1 : 0;
}

// proj fp32 rows of ``stride`` floats [q: heads*d | k: heads*d | v: heads*dv | gate: heads*dv]; decay fp32 [heads]; state
// fp32 [slots, heads, d, dv]; out [tokens, heads*dv] in the storage type; tokens: one per sequence.
CPM_API int cpm_retention_step(const float* proj, int64_t stride, const float* decay, float* state, const int* positions,
                               const int* token_seq, const int* slots, void* out, int n_tokens, int heads, int d, int dv, int rot,
                               const float* inv_freq, float magnitude, int adjacent, float k_factor, float eps, int dtype,
                               cudaStream_t stream) {
    if (n_tokens <= 0) return CPM_OK;
    if (heads < 1 || heads > 65535 || !cpm_retention_step_sizes(d, dv) || rot < 0 || (rot & 1) || rot > d || (rot && !inv_freq) ||
        stride < 2 * (int64_t)heads * (d + dv))
        return CPM_BAD_ARGUMENT;
    const int vec = dv % 4 == 0 ? 4 : 1, rows_at_once = kStepThreads / (dv / vec);
    const size_t smem = (size_t)(2 * d + rows_at_once * dv + dv + 33) * sizeof(float);      // at most 8 + 4 + 4 KiB
    const dim3 grid(n_tokens, heads), block(kStepThreads);
#define CPM_RET_STEP(TT, V)                                                                                                          \
    cpm_launch(kLaunchAttention, retention_step_kernel<TT, V>, grid, block, smem, stream, proj, stride, decay, state, positions,     \
               token_seq, slots, (TT*)out, heads, d, dv, rot, inv_freq, magnitude, adjacent, k_factor, eps)
    if (dtype == CPM_BF16) { if (vec == 4) CPM_RET_STEP(bf16, 4); else CPM_RET_STEP(bf16, 1); }
    else { if (vec == 4) CPM_RET_STEP(float, 4); else CPM_RET_STEP(float, 1); }
#undef CPM_RET_STEP
    return launch_status();
}

// ---------------------------------------------------------------------------
// Prompts: tiles of 64 tokens.
// ---------------------------------------------------------------------------
// The tokens of a tile: [t0, t0 + n) of the step's token axis (n <= 0: an unused tile).
struct RetTile { int seq, t0, n; };
__device__ __forceinline__ RetTile ret_tile(const int* __restrict__ tile_seq, const int* __restrict__ tile_row, const int* __restrict__ cu_q,
                                            int tile) {
    RetTile r;
    r.seq = tile_seq[tile];
    r.t0 = cu_q[r.seq] + tile_row[tile];
    r.n = min(kRetTile, cu_q[r.seq + 1] - r.t0);
    return r;
}

// Four consecutive floats of a row of ``width``, zeros beyond it; ``vec``: rows and width allow one 16-byte load.
__device__ __forceinline__ float4 row4(const float* __restrict__ p, int c, int width, bool vec) {
    if (vec) return c < width ? load4(p + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    return make_float4(c < width ? p[c] : 0.f, c + 1 < width ? p[c + 1] : 0.f, c + 2 < width ? p[c + 2] : 0.f, c + 3 < width ? p[c + 3] : 0.f);
}

// A block: 64 key channels x 64 value columns of one tile's U; a thread 8 x 4 of them.
constexpr int kKvThreads = 128;

__global__ void __launch_bounds__(kKvThreads)
retention_tile_kv_kernel(const float* __restrict__ k, int64_t k_stride, const float* __restrict__ v, int64_t v_stride,
                         const float* __restrict__ powers /* [heads][65] */, const int* __restrict__ tile_seq,
                         const int* __restrict__ tile_row, const int* __restrict__ cu_q, float* __restrict__ U, int heads, int d, int dv,
                         int v_blocks, int vec) {
    __shared__ __align__(16) float ks[kRetTile][kRetPitch];
    __shared__ __align__(16) float vs[kRetTile][kRetPitch];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, c0 = (blockIdx.z / v_blocks) * 64, e0 = (blockIdx.z % v_blocks) * 64;
    const RetTile tl = ret_tile(tile_seq, tile_row, cu_q, blockIdx.x);
    if (tl.n <= 0) return;
    const float* pw = powers + h * (kRetTile + 1);
#pragma unroll 4
    for (int e = threadIdx.x; e < kRetTile * 16; e += kKvThreads) {
        const int j = e >> 4, c = 4 * (e & 15);
        float4 kv = make_float4(0.f, 0.f, 0.f, 0.f), vv = kv;
        if (j < tl.n) {
            kv = row4(k + (int64_t)(tl.t0 + j) * k_stride + (int64_t)h * d, c0 + c, d, vec);
            vv = row4(v + (int64_t)(tl.t0 + j) * v_stride + (int64_t)h * dv, e0 + c, dv, vec);
            const float f = pw[tl.n - 1 - j];
            kv = make_float4(kv.x * f, kv.y * f, kv.z * f, kv.w * f);
        }
        store4(&ks[j][c], kv);
        store4(&vs[j][c], vv);
    }
    __syncthreads();
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[8][4] = {};
#pragma unroll 4
    for (int j = 0; j < kRetTile; ++j) {
        const float4 a = load4(&ks[j][8 * ty]), a2 = load4(&ks[j][8 * ty + 4]), b = load4(&vs[j][4 * tx]);
        const float av[8] = {a.x, a.y, a.z, a.w, a2.x, a2.y, a2.z, a2.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int r = 0; r < 8; ++r)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[r][c] = fmaf(av[r], bv[c], acc[r][c]);
    }
    float* dst = U + ((int64_t)blockIdx.x * heads + h) * d * dv;
#pragma unroll
    for (int r = 0; r < 8; ++r) {
        const int c = c0 + 8 * ty + r, e = e0 + 4 * tx;
        if (c >= d) continue;
        if (vec) {
            if (e < dv) store4(dst + (int64_t)c * dv + e, make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]));
        } else {
#pragma unroll
            for (int x = 0; x < 4; ++x)
                if (e + x < dv) dst[(int64_t)c * dv + e + x] = acc[r][x];
        }
    }
}

constexpr int kScanFlight = 8;       // tiles whose U a thread asks for at a time, one batch ahead of the one it works on

template <int VEC>
__global__ void __launch_bounds__(256)
retention_tile_scan_kernel(float* __restrict__ U, float* __restrict__ state, const float* __restrict__ powers,
                           const int* __restrict__ positions, const int* __restrict__ cu_q, const int* __restrict__ slots, int heads,
                           int64_t elems /* d * dv */) {
    __shared__ int first_tile;
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y, seq = blockIdx.z;
    const int t0 = cu_q[seq], len = cu_q[seq + 1] - t0;
    if (len <= 0) return;
    if (threadIdx.x == 0) first_tile = 0;
    __syncthreads();
    int mine = 0;                                 // tiles of the sequences before this one
    for (int s = threadIdx.x; s < seq; s += blockDim.x) mine += (max(cu_q[s + 1] - cu_q[s], 0) + kRetTile - 1) / kRetTile;
    if (mine) atomicAdd(&first_tile, mine);
    __syncthreads();
    const int64_t e = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (e >= elems) return;
    const float* pw = powers + h * (kRetTile + 1);
    const int n_tiles = (len + kRetTile - 1) / kRetTile;
    const float full = pw[kRetTile], last = pw[len - (n_tiles - 1) * kRetTile];
    float* st = state + ((int64_t)slots[seq] * heads + h) * elems + e;
    float* u0 = U + ((int64_t)first_tile * heads + h) * elems + e;
    const int64_t step = (int64_t)heads * elems;
    float S[VEC];
    const bool fresh = positions[t0] == 0;
#pragma unroll
    for (int j = 0; j < VEC; ++j) S[j] = 0.f;
    if (!fresh) {
        if (VEC == 4) { const float4 f = load4(st); S[0] = f.x; S[1 % VEC] = f.y; S[2 % VEC] = f.z; S[3 % VEC] = f.w; }
        else S[0] = st[0];
    }
    float u[kScanFlight][VEC], next[kScanFlight][VEC];
    auto fetch = [&](float (&to)[kScanFlight][VEC], int i0) {
#pragma unroll
        for (int i = 0; i < kScanFlight; ++i) {
            if (i0 + i < n_tiles) {
                const float* src = u0 + (i0 + i) * step;
                if (VEC == 4) { const float4 f = load4(src); to[i][0] = f.x; to[i][1 % VEC] = f.y; to[i][2 % VEC] = f.z; to[i][3 % VEC] = f.w; }
                else to[i][0] = src[0];
            }
        }
    };
    fetch(u, 0);
    for (int i0 = 0; i0 < n_tiles; i0 += kScanFlight) {
        fetch(next, i0 + kScanFlight);
#pragma unroll
        for (int i = 0; i < kScanFlight; ++i) {
            if (i0 + i < n_tiles) {
                float* dst = u0 + (i0 + i) * step;
                if (VEC == 4) store4(dst, make_float4(S[0], S[1 % VEC], S[2 % VEC], S[3 % VEC]));
                else dst[0] = S[0];
                const float f = i0 + i + 1 < n_tiles ? full : last;
#pragma unroll
                for (int j = 0; j < VEC; ++j) S[j] = fmaf(f, S[j], u[i][j]);
            }
        }
#pragma unroll
        for (int i = 0; i < kScanFlight; ++i)
#pragma unroll
            for (int j = 0; j < VEC; ++j) u[i][j] = next[i][j];
    }
    if (VEC == 4) store4(st, make_float4(S[0], S[1 % VEC], S[2 % VEC], S[3 % VEC]));
    else st[0] = S[0];
}

// A block: the 64 tokens of a tile x all value columns of a head (NC groups of 64); a thread 4 tokens x 4 NC columns
// (4 tx + 64 g).  One walk over the key channels, a slice at a time, gives the scores of all pairs of the tile and the read-out
// of the state before it; then the tile's own keys.  NORM: o / rms(o) * SiLU(gate) in the storage type; else o as it is, fp32
// (T = float).
template <typename T, int NC, bool NORM>
__global__ void __launch_bounds__(256, NC <= 2 ? 3 : 2)
retention_tile_out_kernel(const float* __restrict__ q, const float* __restrict__ k, int64_t qk_stride, const float* __restrict__ v,
                          int64_t v_stride, const float* __restrict__ gate, int64_t gate_stride, const float* __restrict__ powers,
                          const int* __restrict__ tile_seq, const int* __restrict__ tile_row, const int* __restrict__ cu_q,
                          const float* __restrict__ S, T* __restrict__ out, int heads, int d, int dv, float eps, int vec) {
    constexpr int kCols = 64 * NC;
    constexpr int kSlice = NC <= 2 ? 32 : 16;     // key channels, or keys, that are staged at a time
    __shared__ __align__(16) float qk[kRetTile * kRetPitch];        // a slice of queries and of keys, channel by channel
    __shared__ __align__(16) float stage[kSlice * kCols];           // rows of the state, or values
    __shared__ float pw[kRetTile + 1];
    float* qt = qk;
    float* kt = qk + kSlice * kRetPitch;
    float* as = qk;                               // later: decayed scores [64 keys][68 queries]
    static_assert(2 * kSlice <= kRetTile, "the scores take the place of the two slices");
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.y;
    const RetTile tl = ret_tile(tile_seq, tile_row, cu_q, blockIdx.x);
    if (tl.n <= 0) return;
    if (threadIdx.x <= kRetTile) pw[threadIdx.x] = powers[h * (kRetTile + 1) + threadIdx.x];
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const float* qh = q + (int64_t)tl.t0 * qk_stride + (int64_t)h * d;
    const float* kh = k + (int64_t)tl.t0 * qk_stride + (int64_t)h * d;
    const float* vh = v + (int64_t)tl.t0 * v_stride + (int64_t)h * dv;
    const float* Sh = S + ((int64_t)blockIdx.x * heads + h) * d * dv;
    float s[4][4] = {};
    float o[4][4 * NC] = {};
    for (int c0 = 0; c0 < d; c0 += kSlice) {
        if (c0) __syncthreads();
        // a warp takes 4 channels of 32 tokens at a time: its stores into the transposed rows hit 32 different banks
#pragma unroll
        for (int u = warp; u < 2 * (kSlice / 4); u += 8) {
            const int i = (u & 1) * 32 + lane, c = 4 * (u >> 1);
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
            if (i < tl.n) {
                a = row4(qh + (int64_t)i * qk_stride, c0 + c, d, vec);
                b = row4(kh + (int64_t)i * qk_stride, c0 + c, d, vec);
            }
            qt[(c + 0) * kRetPitch + i] = a.x;
            qt[(c + 1) * kRetPitch + i] = a.y;
            qt[(c + 2) * kRetPitch + i] = a.z;
            qt[(c + 3) * kRetPitch + i] = a.w;
            kt[(c + 0) * kRetPitch + i] = b.x;
            kt[(c + 1) * kRetPitch + i] = b.y;
            kt[(c + 2) * kRetPitch + i] = b.z;
            kt[(c + 3) * kRetPitch + i] = b.w;
        }
#pragma unroll
        for (int e = threadIdx.x; e < kSlice * (kCols / 4); e += 256) {
            const int m = e / (kCols / 4), c = 4 * (e % (kCols / 4));
            store4(stage + m * kCols + c, c0 + m < d ? row4(Sh + (int64_t)(c0 + m) * dv, c, dv, vec) : make_float4(0.f, 0.f, 0.f, 0.f));
        }
        __syncthreads();
#pragma unroll 4
        for (int c = 0; c < kSlice; ++c) {
            const float4 a = load4(qt + c * kRetPitch + 4 * ty), b = load4(kt + c * kRetPitch + 4 * tx);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int r = 0; r < 4; ++r)
#pragma unroll
                for (int x = 0; x < 4; ++x) s[r][x] = fmaf(av[r], bv[x], s[r][x]);
#pragma unroll
            for (int g = 0; g < NC; ++g) {
                const float4 z = load4(stage + c * kCols + 64 * g + 4 * tx);
                const float zv[4] = {z.x, z.y, z.z, z.w};
#pragma unroll
                for (int r = 0; r < 4; ++r)
#pragma unroll
                    for (int x = 0; x < 4; ++x) o[r][4 * g + x] = fmaf(av[r], zv[x], o[r][4 * g + x]);
            }
        }
    }
    __syncthreads();                              // the slices are no longer read: the scores take their place
#pragma unroll
    for (int x = 0; x < 4; ++x) {
        float w[4];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
            const int i = 4 * ty + r, j = 4 * tx + x;
            w[r] = j <= i ? s[r][x] * pw[i - j] : 0.f;
        }
        store4(as + (4 * tx + x) * kRetPitch + 4 * ty, make_float4(w[0], w[1], w[2], w[3]));
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        const float f = pw[4 * ty + r + 1];
#pragma unroll
        for (int x = 0; x < 4 * NC; ++x) o[r][x] *= f;
    }
    // the tile's own keys
    for (int j0 = 0; j0 < tl.n; j0 += kSlice) {
        __syncthreads();
        for (int e = threadIdx.x; e < kSlice * (kCols / 4); e += 256) {
            const int m = e / (kCols / 4), c = 4 * (e % (kCols / 4));
            store4(stage + m * kCols + c, j0 + m < tl.n ? row4(vh + (int64_t)(j0 + m) * v_stride, c, dv, vec) : make_float4(0.f, 0.f, 0.f, 0.f));
        }
        __syncthreads();
        const int count = min(kSlice, 8 * warp + 8 - j0);                  // a warp's rows end at 8 warp + 7
#pragma unroll 4
        for (int m = 0; m < count; ++m) {
            const float4 a = load4(as + (j0 + m) * kRetPitch + 4 * ty);
            const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
            for (int g = 0; g < NC; ++g) {
                const float4 b = load4(stage + m * kCols + 64 * g + 4 * tx);
                const float bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
                for (int r = 0; r < 4; ++r)
#pragma unroll
                    for (int x = 0; x < 4; ++x) o[r][4 * g + x] = fmaf(av[r], bv[x], o[r][4 * g + x]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        const int i = 4 * ty + r;
        float f = 1.f;
        if (NORM) {
            float ss = 0.f;                       // columns beyond dv are zero
#pragma unroll
            for (int x = 0; x < 4 * NC; ++x) ss = fmaf(o[r][x], o[r][x], ss);
#pragma unroll
            for (int w = 1; w < 16; w <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
            f = 1.0f / sqrtf(ss / (float)dv + eps);
        }
        if (i >= tl.n) continue;
        T* dst = out + ((int64_t)(tl.t0 + i) * heads + h) * dv;
        const float* gr = NORM ? gate + (int64_t)(tl.t0 + i) * gate_stride + (int64_t)h * dv : nullptr;
#pragma unroll
        for (int g = 0; g < NC; ++g) {
            const int e = 64 * g + 4 * tx;
            if (vec) {
                if (e < dv) {
                    float4 res = make_float4(o[r][4 * g] * f, o[r][4 * g + 1] * f, o[r][4 * g + 2] * f, o[r][4 * g + 3] * f);
                    if (NORM) {
                        const float4 z = load4(gr + e);
                        res = make_float4(res.x * ret_silu(z.x), res.y * ret_silu(z.y), res.z * ret_silu(z.z), res.w * ret_silu(z.w));
                    }
                    store4(dst + e, res);
                }
            } else {
#pragma unroll
                for (int x = 0; x < 4; ++x)
                    if (e + x < dv) dst[e + x] = from_f32<T>(o[r][4 * g + x] * f * (NORM ? ret_silu(gr[e + x]) : 1.f));
            }
        }
    }
}

CPM_API int64_t cpm_retention_tiles_scratch_floats(int n_tiles, int heads, int d, int dv) { return (int64_t)n_tiles * heads * d * dv; }

template <typename T, int NC, bool NORM>
static int launch_tile_out(const float* q, const float* k, int64_t qk_stride, const float* v, int64_t v_stride, const float* gate,
                           int64_t gate_stride, const float* powers, const int* tile_seq, const int* tile_row, int n_tiles,
                           const int* cu_q, const float* S, void* out, int heads, int d, int dv, float eps, int vec,
                           cudaStream_t stream) {
    auto kern = retention_tile_out_kernel<T, NC, NORM>;
    cpm_launch(kLaunchAttention, kern, dim3(n_tiles, heads), dim3(256), 0, stream, q, k, qk_stride, v, v_stride, gate, gate_stride,
               powers, tile_seq, tile_row, cu_q, S, (T*)out, heads, d, dv, eps, vec);
    return launch_status();
}

// q, k: fp32 rows of ``qk_stride`` floats holding [heads, d] (turned, k scaled); v, gate: rows holding [heads, dv]; powers fp32
// [heads, 65]: a_h^0 .. a_h^64; state fp32 [slots, heads, d, dv], read at a sequence's first token of the step (zeros at
// position 0) and written at its last; scratch: cpm_retention_tiles_scratch_floats floats.  The tiles list every sequence's
// tokens in order, sequence after sequence, 64 tokens a tile; tiles behind them belong to an empty sequence.  gate given:
// out [tokens, heads*dv] in the storage type, normed and gated; else fp32 [tokens, heads, dv].
CPM_API int cpm_retention_tiles(const float* q, const float* k, int64_t qk_stride, const float* v, int64_t v_stride, const float* gate,
                                int64_t gate_stride, const float* powers, float* state, const int* positions, const int* cu_q,
                                const int* slots, const int* tile_seq, const int* tile_row, int n_tiles, int n_seqs, float* scratch,
                                void* out, int heads, int d, int dv, float eps, int dtype, cudaStream_t stream) {
    if (n_tiles <= 0 || n_seqs <= 0) return CPM_OK;
    if (heads < 1 || heads > 65535 || n_seqs > 65535 || d < 1 || d > 256 || dv < 1 || dv > 256 || scratch == nullptr) return CPM_BAD_ARGUMENT;
    auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const int vec = d % 4 == 0 && dv % 4 == 0 && qk_stride % 4 == 0 && v_stride % 4 == 0 && gate_stride % 4 == 0 && aligned(q) && aligned(k) &&
                    aligned(v) && (gate == nullptr || aligned(gate));
    const int c_blocks = (d + 63) / 64, v_blocks = (dv + 63) / 64;
    cpm_launch(kLaunchAttention, retention_tile_kv_kernel, dim3(n_tiles, heads, c_blocks * v_blocks), dim3(kKvThreads), 0, stream, k, qk_stride, v,
               v_stride, powers, tile_seq, tile_row, cu_q, scratch, heads, d, dv, v_blocks, vec);
    const int64_t elems = (int64_t)d * dv;
    if (elems % 4 == 0)
        cpm_launch(kLaunchAttention, retention_tile_scan_kernel<4>, dim3((unsigned)((elems / 4 + 255) / 256), heads, n_seqs), dim3(256), 0, stream,
                   scratch, state, powers, positions, cu_q, slots, heads, elems);
    else
        cpm_launch(kLaunchAttention, retention_tile_scan_kernel<1>, dim3((unsigned)((elems + 255) / 256), heads, n_seqs), dim3(256), 0, stream,
                   scratch, state, powers, positions, cu_q, slots, heads, elems);
#define CPM_RET_OUT(TT, N, G) launch_tile_out<TT, N, G>(q, k, qk_stride, v, v_stride, gate, gate_stride, powers, tile_seq, tile_row, n_tiles, \
                                                        cu_q, (const float*)scratch, out, heads, d, dv, eps, vec, stream)
#define CPM_RET_WIDTH(TT, G) (dv <= 64 ? CPM_RET_OUT(TT, 1, G) : dv <= 128 ? CPM_RET_OUT(TT, 2, G) : CPM_RET_OUT(TT, 4, G))
    if (gate == nullptr) return CPM_RET_WIDTH(float, false);
    if (dtype == CPM_BF16) return CPM_RET_WIDTH(bf16, true);
    return CPM_RET_WIDTH(float, true);
#undef CPM_RET_WIDTH
#undef CPM_RET_OUT
}

// Latent attention: the step between the down-projections and the attention over the latent cache.
//
// A token's row of the stacked down-projection holds [a_q (q_rank values) | a_kv (kv_rank values)].
// Both halves are RMS-normed with a weight of their own (float32 arithmetic):
//     c_q = a_q  / sqrt(mean(a_q^2)  + eps) * w_q      -> cq_out [T, q_rank]   (input of the query up-projection)
//     c   = a_kv / sqrt(mean(a_kv^2) + eps) * w_kv     -> cache row `slots[t]` (the only thing kept per token)
// The cache row is `row_width` wide (kv_rank rounded up to what the attention kernels take); the tail is
// written as zeros, so that keys of any rank are plain rows of a one-head cache [pages, 1, page_size, row_width].
// A row may carry a third part behind a_kv: `rot_dim` values that are NOT normed, one rotated key part shared by all
// heads.  Its first `rot` features are turned by the token's position (pairs (i, i + rot/2), angle = (float)pos *
// inv_freq[i], float32, sine and cosine times `amp`) and the part is written into the cache row behind the latent,
// [c | rotated part | zeros].  vl_rope_heads turns the matching part of every query head in place; a design without a query
// latent has its finished query heads in the same row, and then this kernel turns them as well.
// One block of 128 threads per token; the order of every sum depends on the sizes alone.
// A negative slot (a padded token of a graph step) writes no cache row; a slot outside the pool sets
// VL_DEV_BAD_SLOT and is skipped.
#include "common.cuh"

#define LATENT_MAX_PAIRS 256         // most rotated pairs of a head

// sine and cosine (times `amp`) of every pair's angle at this position, made once per token
__device__ __forceinline__ void latent_angles(float2* table, int half, float pos, float amp, const float* __restrict__ inv_freq) {
    for (int i = threadIdx.x; i < half; i += 128) {
        float sn, cs;
        sincosf(pos * inv_freq[i], &sn, &cs);
        table[i] = make_float2(cs * amp, sn * amp);
    }
}
// features [0, rot) of every head turned in place: head h at row + h * stride
template <typename T>
__device__ __forceinline__ void latent_turn(T* row, int stride, int heads, int half, const float2* table) {
    for (int idx = threadIdx.x; idx < heads * half; idx += 128) {
        const int h = idx / half, i = idx - h * half;
        const float2 cs = table[i];
        T* p = row + (size_t)h * stride;
        const float u = to_f32(p[i]), v = to_f32(p[i + half]);
        p[i] = from_f32<T>(u * cs.x - v * cs.y);
        p[i + half] = from_f32<T>(v * cs.x + u * cs.y);
    }
}

// The latent (and the rotated key part) of a row starts at column kv_col.  q_rank > 0: a_q lies at column 0 and is normed into
// cq_out.  q_heads > 0: the row holds finished query heads instead, head h's rotated part at column q_col + h * q_stride,
// which is turned in place.
template <typename T>
__global__ void __launch_bounds__(128)
latent_norm_write_kernel(T* __restrict__ proj, int ld, int q_rank, int kv_col, int kv_rank,
                         const float* __restrict__ wq, const float* __restrict__ wkv, float eps,
                         T* __restrict__ cq_out, const int* __restrict__ slots, T* __restrict__ cache,
                         int row_width, long long num_slots, int rot_dim, int rot, const float* __restrict__ inv_freq, float amp,
                         int q_col, int q_stride, int q_heads, const int* __restrict__ positions, unsigned* err) {
    __shared__ float scratch[32];
    __shared__ float2 table[LATENT_MAX_PAIRS];
    pdl_launch_dependents();
    const int t = blockIdx.x, half = rot / 2;
    if (half > 0) latent_angles(table, half, (float)positions[t], amp, inv_freq);
    pdl_wait();
    T* row = proj + (size_t)t * ld;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < q_rank; i += 128) { const float v = to_f32(row[i]); sq += v * v; }
    for (int i = threadIdx.x; i < kv_rank; i += 128) { const float v = to_f32(row[kv_col + i]); sk += v * v; }
    if (q_rank > 0) sq = block_sum<128>(sq, scratch);
    sk = block_sum<128>(sk, scratch);                            // (its barriers also publish the table)
    const float ik = 1.0f / sqrtf(sk / (float)kv_rank + eps);
    if (q_rank > 0) {
        const float iq = 1.0f / sqrtf(sq / (float)q_rank + eps);
        T* cq = cq_out + (size_t)t * q_rank;
        for (int i = threadIdx.x; i < q_rank; i += 128) cq[i] = from_f32<T>(to_f32(row[i]) * iq * wq[i]);
    }
    if (q_heads > 0 && half > 0) latent_turn(row + q_col, q_stride, q_heads, half, table);
    if (!slots) return;
    const long long slot = slots[t];
    if (slot < 0) return;
    if (slot >= num_slots) {
        if (threadIdx.x == 0) atomicOr(err, VL_DEV_BAD_SLOT);
        return;
    }
    T* dst = cache + (size_t)slot * row_width;
    for (int i = threadIdx.x; i < row_width; i += 128) {
        float v = 0.f;
        if (i < kv_rank) {
            v = to_f32(row[kv_col + i]) * ik * wkv[i];
        } else if (i < kv_rank + rot_dim) {
            const int e = i - kv_rank;
            const T* tail = row + kv_col + kv_rank;
            v = to_f32(tail[e]);
            if (e < rot) {
                const float2 cs = table[e < half ? e : e - half];
                v = e < half ? v * cs.x - to_f32(tail[e + half]) * cs.y : v * cs.x + to_f32(tail[e - half]) * cs.y;
            }
        }
        dst[i] = from_f32<T>(v);
    }
}

// The same with eight neighbouring numbers a thread (16-byte accesses in bfloat16), where every part of a row starts on such a
// boundary: the ranks, the columns, the rotated half and the heads' stride are multiples of 8.
template <typename T>
__global__ void __launch_bounds__(128)
latent_norm_write_vec_kernel(T* __restrict__ proj, int ld, int q_rank, int kv_col, int kv_rank,
                             const float* __restrict__ wq, const float* __restrict__ wkv, float eps,
                             T* __restrict__ cq_out, const int* __restrict__ slots, T* __restrict__ cache,
                             int row_width, long long num_slots, int rot_dim, int rot, const float* __restrict__ inv_freq, float amp,
                             int q_col, int q_stride, int q_heads, const int* __restrict__ positions, unsigned* err) {
    __shared__ float scratch[32];
    __shared__ float2 table[LATENT_MAX_PAIRS];
    pdl_launch_dependents();
    const int t = blockIdx.x, half = rot / 2, tid = threadIdx.x;
    if (half > 0) latent_angles(table, half, (float)positions[t], amp, inv_freq);
    pdl_wait();
    T* row = proj + (size_t)t * ld;
    float sq = 0.f, sk = 0.f, a[8], c[8];
    for (int i = 8 * tid; i < q_rank; i += 1024) {
        load8(row + i, a);
#pragma unroll
        for (int e = 0; e < 8; ++e) sq += a[e] * a[e];
    }
    const bool latent = 8 * tid < kv_rank;                       // (a row's latent fits one piece a thread: at most 1,024 numbers)
    if (latent) {
        load8(row + kv_col + 8 * tid, c);
#pragma unroll
        for (int e = 0; e < 8; ++e) sk += c[e] * c[e];
    }
    if (q_rank > 0) sq = block_sum<128>(sq, scratch);
    sk = block_sum<128>(sk, scratch);                            // (its barriers also publish the table)
    if (q_rank > 0) {
        const float iq = 1.0f / sqrtf(sq / (float)q_rank + eps);
        for (int i = 8 * tid; i < q_rank; i += 1024) {           // (one piece a thread up to 1,024 numbers: still in registers)
            if (q_rank > 1024) load8(row + i, a);
#pragma unroll
            for (int e = 0; e < 8; ++e) a[e] *= iq * wq[i + e];
            store8(cq_out + (size_t)t * q_rank + i, a);
        }
    }
    const int pieces = half / 8;
    for (int idx = tid; idx < q_heads * pieces; idx += 128) {
        const int h = idx / pieces, i = 8 * (idx - h * pieces);
        T* p = row + q_col + (size_t)h * q_stride + i;
        float u[8], v[8];
        load8(p, u);
        load8(p + half, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
            const float2 cs = table[i + e];
            const float x = u[e], y = v[e];
            u[e] = x * cs.x - y * cs.y;
            v[e] = y * cs.x + x * cs.y;
        }
        store8(p, u);
        store8(p + half, v);
    }
    if (!slots) return;
    const long long slot = slots[t];
    if (slot < 0) return;
    if (slot >= num_slots) {
        if (tid == 0) atomicOr(err, VL_DEV_BAD_SLOT);
        return;
    }
    T* dst = cache + (size_t)slot * row_width;
    if (latent) {
        const float ik = 1.0f / sqrtf(sk / (float)kv_rank + eps);
#pragma unroll
        for (int e = 0; e < 8; ++e) c[e] *= ik * wkv[8 * tid + e];
        store8(dst + 8 * tid, c);
    }
    for (int i = kv_rank + 8 * tid; i < row_width; i += 1024) {
        const int e0 = i - kv_rank;
        const T* tail = row + kv_col + kv_rank;
        float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (e0 < rot_dim) {
            load8(tail + e0, v);
            if (e0 < rot) {
                const bool low = e0 < half;
                float o[8];
                load8(tail + (low ? e0 + half : e0 - half), o);
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    const float2 cs = table[(low ? e0 : e0 - half) + e];
                    v[e] = low ? v[e] * cs.x - o[e] * cs.y : v[e] * cs.x + o[e] * cs.y;
                }
            }
        }
        store8(dst + i, v);
    }
}

// x [T, ld]: for every head h < heads the features col0 + h * stride + [0, rot) are turned in place by the token's
// position (rotate-half pairs, float32 angles, sine and cosine times amp).  A block per token, a thread per (head, pair).
template <typename T>
__global__ void __launch_bounds__(128)
rope_heads_kernel(T* __restrict__ x, int ld, int col0, int stride, int heads, int rot, const float* __restrict__ inv_freq, float amp,
                  const int* __restrict__ positions) {
    __shared__ float2 table[LATENT_MAX_PAIRS];
    pdl_launch_dependents();
    const int t = blockIdx.x, half = rot / 2;
    latent_angles(table, half, (float)positions[t], amp, inv_freq);
    __syncthreads();
    pdl_wait();
    latent_turn(x + (size_t)t * ld + col0, stride, heads, half, table);
}

extern "C" int vl_rope_heads(void* x, int dtype, int T, int ld, int col0, int stride, int heads, int rot, const float* inv_freq,
                             float amp, const int* positions, void* stream) {
    if (T <= 0 || rot <= 0) return VL_OK;
    if ((rot & 1) || heads <= 0 || stride < rot || col0 < 0 || col0 + (heads - 1) * stride + rot > ld || !inv_freq || !positions)
        return VL_ERR_ARGUMENT;
    if (rot / 2 > LATENT_MAX_PAIRS) return VL_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == VL_F32)
        return vl_launch(rope_heads_kernel<float>, dim3(T), dim3(128), 0, s, (float*)x, ld, col0, stride, heads, rot, inv_freq, amp, positions);
    if (dtype == VL_BF16)
        return vl_launch(rope_heads_kernel<bf16>, dim3(T), dim3(128), 0, s, (bf16*)x, ld, col0, stride, heads, rot, inv_freq, amp, positions);
    return VL_ERR_UNSUPPORTED;
}

extern "C" int vl_latent_norm_write(void* proj, int dtype, int ld, int T, int q_rank, int kv_col, int kv_rank,
                                    const float* wq, const float* wkv, float eps, void* cq_out,
                                    const int* slots, void* cache, int row_width, long long num_slots,
                                    int rot_dim, int rot, const float* inv_freq, float amp, int q_col, int q_stride, int q_heads,
                                    const int* positions, unsigned* err, void* stream) {
    if (T <= 0) return VL_OK;
    if (q_rank < 0 || kv_rank <= 0 || rot_dim < 0 || kv_col < q_rank || ld < kv_col + kv_rank + rot_dim || row_width < kv_rank + rot_dim)
        return VL_ERR_ARGUMENT;
    if (rot < 0 || (rot & 1) || rot > rot_dim || (rot > 0 && (!inv_freq || !positions)) || (q_rank > 0 && (!wq || !cq_out)))
        return VL_ERR_ARGUMENT;
    if (q_heads < 0 || (q_heads > 0 && (q_col < 0 || q_stride < rot || q_col + (long long)(q_heads - 1) * q_stride + rot > kv_col)))
        return VL_ERR_ARGUMENT;
    if (rot / 2 > LATENT_MAX_PAIRS) return VL_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    // (float32 steps keep the one form whose sums do not depend on such boundaries)
    const bool vec = dtype == VL_BF16 && ((ld | q_rank | kv_col | kv_rank | row_width | rot_dim | (rot / 2) | (q_heads > 0 ? q_col | q_stride : 0)) & 7) == 0 &&
                     kv_rank <= 1024 && (((uintptr_t)proj | (uintptr_t)cq_out | (uintptr_t)cache) & 15) == 0;
#define LATENT_WRITE(KERNEL, TT)                                                                                                             \
    return vl_launch(KERNEL<TT>, dim3(T), dim3(128), 0, s, (TT*)proj, ld, q_rank, kv_col, kv_rank, wq, wkv, eps,   \
                     (TT*)cq_out, slots, (TT*)cache, row_width, num_slots, rot_dim, rot, inv_freq, amp, q_col, q_stride, q_heads,    \
                     positions, err)
    if (dtype == VL_F32) LATENT_WRITE(latent_norm_write_kernel, float);
    if (vec) LATENT_WRITE(latent_norm_write_vec_kernel, bf16);
    if (dtype == VL_BF16) LATENT_WRITE(latent_norm_write_kernel, bf16);
#undef LATENT_WRITE
    return VL_ERR_UNSUPPORTED;
}

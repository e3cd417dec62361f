// The head work of an attention in one pass over the product's rows: bias, norm, rotation, a factor per query head, the
// rows of q laid out for the attention kernels and the new keys and values written into the paged cache.
//
// A row of `in` [T, ld] is  q (nq heads x M maps x D) | k (nkv x M x D) | v (nkv x V)  (k and v absent: a call that reads
// another call's cache); `bias` (or null) has an entry per column.  D and V are multiples of 8; what pads a head of another
// size to D is zero and stays zero, the means divide by the true counts (`unit_n` features of a head, `q_n` and `k_n` of a row).
//   norm      a "unit" is one map of one head.  per unit: u <- u / sqrt(sum u^2 / unit_n + eps) * w[D]; or over the whole
//             projection at once (WHOLE): q <- q / sqrt(sum q^2 / q_n + eps) * qw[nq M D], k likewise; or none (qw null)
//   rotation  neighbours (2i, 2i + 1) of the first `rot` features of every unit turn by position * inv_freq[i]
//   factor    query head h times q_factor[h] (or null)
//   q_out [T, nq * M, P]: map m of head h is row h * M + m and holds its D features at m * D .. and zeros elsewhere, so that
//             its product with a cached key row [k_1 | .. | k_M | zeros] (P wide) is the product with that head's map m alone
//             and all maps of a head read one row of keys and one of values;
//   cache     kcache / vcache [pages, nkv, page_size, P] at the token's slot: [k_1 | .. | k_M | zeros], [v | zeros].
// Everything between load and store is float32, so are positions, angles, sine and cosine.  A unit's sum of squares is
// taken by a butterfly over its lanes, a row's by the block: the order depends on the sizes alone.
#include "common.cuh"

#define HW_MAX_ROT 512

template <typename T>
struct HeadWork {
    const T* in; int ld; const float* bias;
    const int* positions; const int* slots;
    const float* qw; const float* kw; float eps; int unit_n, q_n, k_n;
    const float* inv_freq; int rot;
    const float* q_factor;
    T* q_out; T* kcache; T* vcache;
    int nq, nkv, M, D, V, P, has_kv, page_size; long long num_slots; unsigned* err;
};

// eight neighbouring columns of a row, the bias added
template <typename T>
__device__ __forceinline__ void hw_load(const HeadWork<T>& a, const T* row, int col, float (&v)[8]) {
    load8(row + col, v);
    if (a.bias) {
        float b[8];
        load8(a.bias + col, b);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] += b[i];
    }
}
// norm scale and weight, rotation of pairs (the chunk starts at feature f of its unit), factor
__device__ __forceinline__ void hw_finish(float (&v)[8], float inv, const float* w, int f, int rot, const float* s_cos,
                                          const float* s_sin, float factor) {
    if (w) {
        float g[8];
        load8(w, g);
#pragma unroll
        for (int i = 0; i < 8; ++i) v[i] *= inv * g[i];
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        if (f + 2 * j < rot) {
            const float c = s_cos[(f >> 1) + j], s = s_sin[(f >> 1) + j], x = v[2 * j], y = v[2 * j + 1];
            v[2 * j] = x * c - y * s;
            v[2 * j + 1] = y * c + x * s;
        }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= factor;
}
template <typename T>
__device__ __forceinline__ void hw_zero(T* p) {
    const float z[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    store8(p, z);
}
// the cache rows of a token, or -1: nothing to write
template <typename T>
__device__ __forceinline__ long long hw_slot(const HeadWork<T>& a, int t, bool first) {
    const int slot = (a.slots && a.has_kv) ? a.slots[t] : -1;
    if (slot < 0) return -1;
    if ((long long)slot >= a.num_slots) {
        if (first) atomicOr(a.err, VL_DEV_BAD_SLOT);
        return -1;
    }
    return slot;
}
template <typename T>
__device__ __forceinline__ T* hw_cache_row(const HeadWork<T>& a, T* cache, long long slot, int g) {
    const long long page = slot / a.page_size, off = slot - page * a.page_size;
    return cache + ((page * a.nkv + g) * a.page_size + off) * a.P;
}

// ---- a norm per unit (or none): `lanes` lanes (a power of two) share a unit, a lane holds 8 neighbouring features ----
#define HW_THREADS 128
template <typename T>
__global__ void __launch_bounds__(HW_THREADS)
head_work_units_kernel(HeadWork<T> a, int lanes, int units_per_block) {
    __shared__ float s_cos[HW_MAX_ROT / 2], s_sin[HW_MAX_ROT / 2];
    pdl_launch_dependents();
    const int t = blockIdx.x, tid = threadIdx.x;
    const int pos = a.positions[t];
    if (a.inv_freq)
        for (int i = tid; i < a.rot / 2; i += HW_THREADS) sincosf((float)pos * a.inv_freq[i], &s_sin[i], &s_cos[i]);
    pdl_wait();
    __syncthreads();
    const long long slot = hw_slot(a, t, tid == 0 && blockIdx.y == 0);
    const int nQ = a.nq * a.M, nK = a.has_kv ? a.nkv * a.M : 0, nV = a.has_kv ? a.nkv : 0;
    const int units = nQ + (slot >= 0 ? nK + nV : 0);
    const int lo = blockIdx.y * units_per_block, hi = min(units, lo + units_per_block);
    const int sub = tid / lanes, l = tid % lanes, per_pass = HW_THREADS / lanes;
    const T* row = a.in + (size_t)t * a.ld;
    const int rot = a.inv_freq ? a.rot : 0;
    for (int base = lo; base < hi; base += 2 * per_pass) {           // two units a lane in flight
        float v[2][8];
        int col[2], width[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int unit = base + u * per_pass + sub;
            width[u] = unit >= hi ? 0 : (unit < nQ + nK ? a.D : a.V);
            col[u] = unit < nQ + nK ? unit * a.D : (nQ + nK) * a.D + (unit - nQ - nK) * a.V;
#pragma unroll
            for (int i = 0; i < 8; ++i) v[u][i] = 0.f;
            if (8 * l < width[u]) hw_load(a, row, col[u] + 8 * l, v[u]);
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int unit = base + u * per_pass + sub;
            float ss = 0.f;
#pragma unroll
            for (int i = 0; i < 8; ++i) ss += v[u][i] * v[u][i];
            for (int o = 1; o < lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            if (width[u] == 0) continue;
            const bool is_q = unit < nQ, is_k = !is_q && unit < nQ + nK;
            T* dst;
            int at = 0, zero_to;                                    // the unit's features lie at dst + at; zeros from the end of them
            if (is_q) {
                dst = a.q_out + ((size_t)t * nQ + unit) * a.P;
                at = (unit % a.M) * a.D;
                zero_to = a.P;
                for (int c = 8 * l; c < at; c += 8 * lanes) hw_zero(dst + c);
            } else if (is_k) {
                const int g = (unit - nQ) / a.M, m = (unit - nQ) % a.M;
                dst = hw_cache_row(a, a.kcache, slot, g);
                at = m * a.D;
                zero_to = m + 1 == a.M ? a.P : 0;                   // the last map also clears what is behind it
            } else {
                dst = hw_cache_row(a, a.vcache, slot, unit - nQ - nK);
                zero_to = a.P;
            }
            if (8 * l < width[u]) {
                if (is_q || is_k)
                    hw_finish(v[u], a.qw ? 1.0f / sqrtf(ss / (float)a.unit_n + a.eps) : 1.f, a.qw ? (is_q ? a.qw : a.kw) + 8 * l : nullptr,
                              8 * l, rot, s_cos, s_sin, is_q && a.q_factor ? a.q_factor[unit / a.M] : 1.f);
                store8(dst + at + 8 * l, v[u]);
            }
            for (int c = at + width[u] + 8 * l; c < zero_to; c += 8 * lanes) hw_zero(dst + c);
        }
    }
}

// ---- one norm over all of q and one over all of k (M = 1): a block per token ----
template <typename T, int NT>
__global__ void __launch_bounds__(NT)
head_work_rows_kernel(HeadWork<T> a) {
    __shared__ float s_cos[HW_MAX_ROT / 2], s_sin[HW_MAX_ROT / 2];
    __shared__ float scratch[32];
    pdl_launch_dependents();
    const int t = blockIdx.x, tid = threadIdx.x;
    const int pos = a.positions[t];
    if (a.inv_freq)
        for (int i = tid; i < a.rot / 2; i += NT) sincosf((float)pos * a.inv_freq[i], &s_sin[i], &s_cos[i]);
    pdl_wait();
    const long long slot = hw_slot(a, t, tid == 0);
    const T* row = a.in + (size_t)t * a.ld;
    const int rot = a.inv_freq ? a.rot : 0;
    const int Cq = a.nq * a.D, Ck = slot >= 0 ? a.nkv * a.D : 0, Cv = slot >= 0 ? a.nkv * a.V : 0;
    float ssq = 0.f, ssk = 0.f;
    for (int c = 8 * tid; c < Cq + Ck; c += 8 * NT) {
        float v[8], s = 0.f;
        hw_load(a, row, c, v);
#pragma unroll
        for (int i = 0; i < 8; ++i) s += v[i] * v[i];
        if (c < Cq) ssq += s; else ssk += s;
    }
    ssq = block_sum<NT>(ssq, scratch);
    ssk = block_sum<NT>(ssk, scratch);                              // (block_sum's barriers order the table above, too)
    const float invq = 1.0f / sqrtf(ssq / (float)a.q_n + a.eps), invk = 1.0f / sqrtf(ssk / (float)a.k_n + a.eps);
    for (int c = 8 * tid; c < Cq + Ck; c += 8 * NT) {
        float v[8];
        hw_load(a, row, c, v);
        const bool is_q = c < Cq;
        const int e = is_q ? c : c - Cq, h = e / a.D, f = e - h * a.D;
        hw_finish(v, is_q ? invq : invk, (is_q ? a.qw : a.kw) + e, f, rot, s_cos, s_sin, is_q && a.q_factor ? a.q_factor[h] : 1.f);
        T* dst = is_q ? a.q_out + ((size_t)t * a.nq + h) * a.P : hw_cache_row(a, a.kcache, slot, h);
        store8(dst + f, v);
        if (f + 8 == a.D)
            for (int z = a.D; z < a.P; z += 8) hw_zero(dst + z);
    }
    for (int c = 8 * tid; c < Cv; c += 8 * NT) {
        float v[8];
        const int at = Cq + Ck + c, g = c / a.V, f = c - g * a.V;
        hw_load(a, row, at, v);
        T* dst = hw_cache_row(a, a.vcache, slot, g);
        store8(dst + f, v);
        if (f + 8 == a.V)
            for (int z = a.V; z < a.P; z += 8) hw_zero(dst + z);
    }
}

template <typename T>
static int launch_head_work(const HeadWork<T>& a, int T_, int whole, cudaStream_t s) {
    if (whole) {
        // threads by the row's length alone, so that the order of the sums is a matter of the model's sizes
        const int C = a.nq * a.D + (a.has_kv ? a.nkv * (a.D + a.V) : 0);
        if (C > 4096) return vl_launch(head_work_rows_kernel<T, 512>, dim3(T_), dim3(512), 0, s, a);
        if (C > 1024) return vl_launch(head_work_rows_kernel<T, 256>, dim3(T_), dim3(256), 0, s, a);
        return vl_launch(head_work_rows_kernel<T, 128>, dim3(T_), dim3(128), 0, s, a);
    }
    int lanes = 1;
    while (lanes * 8 < a.D || (a.has_kv && lanes * 8 < a.V)) lanes <<= 1;
    const int units = a.nq * a.M + (a.has_kv ? a.nkv * (a.M + 1) : 0), pass = 2 * (HW_THREADS / lanes);
    // few tokens: a pass a block, so that a decode step fills the SMs; many: a block walks all units of its token and makes
    // the table of angles once
    const int per_block = T_ >= 256 ? units : pass;
    return vl_launch(head_work_units_kernel<T>, dim3(T_, (units + per_block - 1) / per_block), dim3(HW_THREADS), 0, s, a, lanes, per_block);
}

extern "C" int vl_head_work(const void* in, int ld, int dtype, const float* bias, const int* positions, const int* slots,
                            const float* qw, const float* kw, float eps, int whole, int unit_n, int q_n, int k_n,
                            const float* inv_freq, int rot, const float* q_factor, void* q_out, void* kcache, void* vcache,
                            int T, int nq, int nkv, int M, int D, int V, int P, int has_kv, int page_size, long long num_slots,
                            unsigned* err, void* stream) {
    if (T <= 0) return VL_OK;
    if (nq <= 0 || nkv <= 0 || M <= 0 || D <= 0 || V <= 0 || D % 8 || V % 8 || P % 8 || D > 256 || V > 256) return VL_ERR_UNSUPPORTED;
    if (P < M * D || P < V || rot < 0 || rot > D || (rot & 1) || rot > HW_MAX_ROT) return VL_ERR_UNSUPPORTED;
    if (ld % 8 || ld < nq * M * D + (has_kv ? nkv * (M * D + V) : 0) || page_size <= 0 || (qw == nullptr) != (kw == nullptr)) return VL_ERR_ARGUMENT;
    if (whole && (M != 1 || !qw || q_n <= 0 || k_n <= 0)) return VL_ERR_ARGUMENT;
    if (!whole && qw && unit_n <= 0) return VL_ERR_ARGUMENT;
    if (((uintptr_t)in | (uintptr_t)q_out | (uintptr_t)kcache | (uintptr_t)vcache | (uintptr_t)bias | (uintptr_t)qw | (uintptr_t)kw) & 15)
        return VL_ERR_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
#define HW_LAUNCH(TT)                                                                                                        \
    do {                                                                                                                     \
        const HeadWork<TT> a = {(const TT*)in, ld, bias, positions, slots, qw, kw, eps, unit_n, q_n, k_n, inv_freq,          \
                                inv_freq ? rot : 0, q_factor, (TT*)q_out, (TT*)kcache, (TT*)vcache, nq, nkv, M, D, V, P,     \
                                has_kv, page_size, num_slots, err};                                                          \
        return launch_head_work<TT>(a, T, whole, s);                                                                         \
    } while (0)
    if (dtype == VL_F32) HW_LAUNCH(float);
    if (dtype == VL_BF16) HW_LAUNCH(bf16);
#undef HW_LAUNCH
    return VL_ERR_UNSUPPORTED;
}

// ---------------------------------------------------------------------------------------------------------
// Two attention maps of every head combined:  o = a_1 - lambda a_2,  o <- o / sqrt(sum o^2 / n + eps) * factor,
// a [T, 2 nq, P] (map m of head h in row 2 h + m), out [T, nq, V]; V a multiple of 8, the features from n on are zero.
// `lanes` lanes share a head, 8 neighbouring features each.
// ---------------------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(HW_THREADS)
combine_maps_kernel(const T* __restrict__ a, T* __restrict__ out, float lambda, float factor, float eps, int n, int P, int V,
                    int lanes, size_t heads) {
    pdl_launch_dependents();
    pdl_wait();
    const int l = threadIdx.x % lanes;
    const size_t h = (size_t)blockIdx.x * (HW_THREADS / lanes) + threadIdx.x / lanes;
    const bool live = h < heads && 8 * l < V;
    float x[8], y[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] = y[i] = 0.f;
    if (live) {
        load8(a + (2 * h) * P + 8 * l, x);
        load8(a + (2 * h + 1) * P + 8 * l, y);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) { x[i] -= lambda * y[i]; ss += x[i] * x[i]; }
    for (int o = 1; o < lanes; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!live) return;
    const float f = factor / sqrtf(ss / (float)n + eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] *= f;
    store8(out + h * V + 8 * l, x);
}

extern "C" int vl_combine_maps(const void* a, void* out, int dtype, float lambda, float factor, float eps, int n, long long heads,
                               int P, int V, void* stream) {
    if (heads <= 0) return VL_OK;
    if (V <= 0 || V % 8 || V > 256 || P < V || P % 8 || n <= 0 || n > V) return VL_ERR_UNSUPPORTED;
    if (((uintptr_t)a | (uintptr_t)out) & 15) return VL_ERR_ARGUMENT;
    int lanes = 1;
    while (lanes * 8 < V) lanes <<= 1;
    const int per = HW_THREADS / lanes;
    const dim3 grid((unsigned)((heads + per - 1) / per));
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == VL_F32)
        return vl_launch(combine_maps_kernel<float>, grid, dim3(HW_THREADS), 0, s, (const float*)a, (float*)out, lambda, factor, eps, n, P, V, lanes, (size_t)heads);
    if (dtype == VL_BF16)
        return vl_launch(combine_maps_kernel<bf16>, grid, dim3(HW_THREADS), 0, s, (const bf16*)a, (bf16*)out, lambda, factor, eps, n, P, V, lanes, (size_t)heads);
    return VL_ERR_UNSUPPORTED;
}

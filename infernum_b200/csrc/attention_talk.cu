// Attention whose heads exchange their scores before the softmax, over the paged cache, and the
// pass that prepares its queries, keys and values.
//
// With H query heads over G key/value heads (head a reads key/value head a / (H / G)):
//
//   s_h(i, j) = sum_g talk[h, g] (q_g(i) . k_g(j))    (all H heads, across key/value heads)
//   o_h(i)    = sum_j softmax_j(s_h(i, .)) v_h(j) * sigmoid(gate_h(i))
//
// Query i sees keys j <= i; with `chunk` > 0 only those of its own run of `chunk` positions
// (floor(j / chunk) = floor(i / chunk), counted from the sequence's position 0), and with
// `window` > 0 only the last `window` of them.
//
//   qk_row_norm_append  rows [q : H d | k : G d | v : G e | ...] as projected: all of q is divided by
//                       its one root mean square and multiplied by a weight of H d values, k likewise
//                       (each when it has a weight); then the first rd dimensions of every head are
//                       rotated (element i with i + rd/2, angle = position * f_i); query head h is
//                       multiplied by q_scale[h] (what scales its scores).  Queries are
//                       written back in place, keys and values to their pages.  32-bit, one rounding.
//                       The values may also be the keys as they were projected.
//   attention_talk      one CTA per row, all heads: keys in tiles of 32 that start at absolute
//                       multiples of 32; the heads' scores, their combination, the running softmax
//                       and the weighted values each a pass over shared memory.  32-bit throughout:
//                       the attention of the 32-bit engine and of sizes without a tensor-core variant.
#include "common.cuh"

using namespace ib;

template <typename T, typename TW>
__global__ void qk_row_norm_append_kernel(T* __restrict__ x, int x_stride, const TW* __restrict__ qw,
                                          const TW* __restrict__ kw, float eps, const float* __restrict__ q_scale,
                                          const float* __restrict__ inv_freq,
                                          int rd, const int* __restrict__ positions, const int* __restrict__ row_entry,
                                          const int* __restrict__ block_tables, int max_blocks, T* __restrict__ k_pool,
                                          T* __restrict__ v_pool, int nh, int nkv, int d, int e, int v_off, int page_size,
                                          int num_pages, unsigned* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    __shared__ float scratch[33];
    const int row = blockIdx.x;
    T* xr = x + (size_t)row * x_stride;
    const int qc = nh * d, kc = nkv * d;
    float fq = 1.f, fk = 1.f;
    if (qw || kw) {
        float sq = 0.f, sk = 0.f;
        for (int c = threadIdx.x; c < qc + kc; c += blockDim.x) {
            const float v = to_f32(xr[c]);
            if (c < qc) sq = fmaf(v, v, sq); else sk = fmaf(v, v, sk);
        }
        sq = block_sum(sq, scratch);
        __syncthreads();
        sk = block_sum(sk, scratch);
        if (qw) fq = 1.f / sqrtf(sq / (float)qc + eps);
        if (kw) fk = 1.f / sqrtf(sk / (float)kc + eps);
    }
    const int pos = positions[row], blk = pos / page_size;
    const int page = blk < max_blocks ? block_tables[(size_t)row_entry[row] * max_blocks + blk] : -1;
    const bool bad = page < 0 || page >= num_pages;
    if (bad && threadIdx.x == 0) atomicOr(err, IB_FLAG_BAD_PAGE);
    const size_t at = bad ? 0 : ((size_t)page * nkv) * page_size + (pos % page_size);  // + g * page_size: a head's row
    const int half = rd >> 1, per_head = d - half;  // a rotated pair is one item
    const int items = (nh + nkv) * per_head + nkv * e;
    for (int it = threadIdx.x; it < items; it += blockDim.x) {
        if (it >= (nh + nkv) * per_head) {
            const int c = it - (nh + nkv) * per_head, g = c / e;
            if (!bad) v_pool[(at + (size_t)g * page_size) * e + c % e] = xr[v_off + c];
            continue;
        }
        const int head = it / per_head, i = it % per_head;
        const bool is_q = head < nh;
        const int base = head * d;  // (keys follow the queries)
        const float f = is_q ? fq * (q_scale ? q_scale[head] : 1.f) : fk;
        const TW* w = is_q ? (qw ? qw + base : nullptr) : (kw ? kw + base - qc : nullptr);
        T* dst = is_q ? xr + base : k_pool + (at + (size_t)(head - nh) * page_size) * d;
        if (!is_q && bad) continue;
        if (i < half) {
            const float a = to_f32(xr[base + i]) * f * (w ? to_f32(w[i]) : 1.f);
            const float b = to_f32(xr[base + i + half]) * f * (w ? to_f32(w[i + half]) : 1.f);
            float sn, cs;
            sincosf((float)pos * inv_freq[i], &sn, &cs);
            dst[i] = from_f32<T>(a * cs - b * sn);
            dst[i + half] = from_f32<T>(b * cs + a * sn);
        } else {
            const int c = i + half;
            dst[c] = from_f32<T>(to_f32(xr[base + c]) * f * (w ? to_f32(w[c]) : 1.f));
        }
    }
}

__device__ __forceinline__ void unpack8(const uint4& raw, float (&v)[8]) {
    const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(p[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ uint4 pack8(const float (&v)[8]) {
    uint4 raw;
    __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) p[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    return raw;
}
__device__ __forceinline__ void load8(const bf16* p, float (&v)[8]) { unpack8(*reinterpret_cast<const uint4*>(p), v); }
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(p);
    *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(p + 4);
}

// The same on bf16 rows, 16 bytes at a time (d, e, rd / 2 and the row stride multiples of 8, 16-byte aligned
// bases).  An item is 8 pairs that are rotated, 8 elements that are not, or 8 elements of a value; every
// thread holds the first ROW_HOLD of its items in registers from the sums to the stores.  The row is asked
// for first; its sines, cosines and place in the pools are worked out (by the last threads, which have the
// fewest items) while it comes.
constexpr int ROW_MAX_PAIRS = 256, ROW_HOLD = 3;

template <typename TW>
__global__ void __launch_bounds__(256, 4)
qk_row_norm_append_vec8_kernel(bf16* __restrict__ x, int x_stride, const TW* __restrict__ qw, const TW* __restrict__ kw,
                               float eps, const float* __restrict__ q_scale, const float* __restrict__ inv_freq, int rd,
                               const int* __restrict__ positions, const int* __restrict__ row_entry,
                               const int* __restrict__ block_tables, int max_blocks, bf16* __restrict__ k_pool,
                               bf16* __restrict__ v_pool, int nh, int nkv, int d, int e, int v_off, int page_size, int num_pages,
                               unsigned* __restrict__ err) {
    pdl_trigger();
    __shared__ __align__(16) float sn_s[ROW_MAX_PAIRS];
    __shared__ __align__(16) float cs_s[ROW_MAX_PAIRS];
    __shared__ float part[2][8];
    __shared__ long long at_s;  // the row's place among all rows of a pool (key/value head 0), -1: none
    const int row = blockIdx.x;
    const int pos = positions[row], entry = row_entry[row];
    const int qc = nh * d, kc = nkv * d, half = rd >> 1;
    const int rot = half >> 3, per_head = rot + ((d - rd) >> 3);
    const int n_qk = (nh + nkv) * per_head, n_all = n_qk + nkv * (e >> 3);
    bf16* xr = x + (size_t)row * x_stride;
    // the first element of item `it` of a head (c), and the head (-1: it is one of the values', c counts from theirs)
    auto place = [&](int it, int& head, int& c) {
        if (it >= n_qk) {
            head = -1;
            c = (it - n_qk) << 3;
        } else {
            head = it / per_head;
            const int p = it - head * per_head;
            c = p < rot ? p << 3 : rd + ((p - rot) << 3);
        }
    };
    int head_of[ROW_HOLD], c_of[ROW_HOLD];
#pragma unroll
    for (int n = 0; n < ROW_HOLD; ++n) place(threadIdx.x + n * blockDim.x, head_of[n], c_of[n]);
    pdl_wait();

    auto squares = [&](int head, int c, const uint4& a4, const uint4& b4, float& sq, float& sk) {
        float v[8], ss = 0.f;
        unpack8(a4, v);
#pragma unroll
        for (int i = 0; i < 8; ++i) ss = fmaf(v[i], v[i], ss);
        if (c < half) {
            unpack8(b4, v);
#pragma unroll
            for (int i = 0; i < 8; ++i) ss = fmaf(v[i], v[i], ss);
        }
        if (head < nh) sq += ss; else sk += ss;
    };
    uint4 ha[ROW_HOLD], hb[ROW_HOLD];
#pragma unroll
    for (int n = 0; n < ROW_HOLD; ++n) {
        if (threadIdx.x + n * blockDim.x >= n_all) break;
        ha[n] = *reinterpret_cast<const uint4*>(xr + (head_of[n] < 0 ? v_off : head_of[n] * d) + c_of[n]);
        if (head_of[n] >= 0 && c_of[n] < half) hb[n] = *reinterpret_cast<const uint4*>(xr + head_of[n] * d + c_of[n] + half);
    }
    {
        const int back = blockDim.x - 1 - threadIdx.x;
        if (back == 0) {
            const int blk = pos / page_size;
            const int page = blk < max_blocks ? block_tables[(size_t)entry * max_blocks + blk] : -1;
            const bool bad = page < 0 || page >= num_pages;
            if (bad) atomicOr(err, IB_FLAG_BAD_PAGE);
            at_s = bad ? -1 : (long long)page * nkv * page_size + pos % page_size;
        }
        for (int j = back; j < half; j += blockDim.x) sincosf((float)pos * inv_freq[j], &sn_s[j], &cs_s[j]);
    }
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int n = 0; n < ROW_HOLD; ++n)
        if (threadIdx.x + n * blockDim.x < n_qk) squares(head_of[n], c_of[n], ha[n], hb[n], sq, sk);
    for (int it = threadIdx.x + ROW_HOLD * blockDim.x; it < n_qk; it += blockDim.x) {
        int head, c;
        place(it, head, c);
        const uint4 a4 = *reinterpret_cast<const uint4*>(xr + head * d + c);
        const uint4 b4 = c < half ? *reinterpret_cast<const uint4*>(xr + head * d + c + half) : make_uint4(0, 0, 0, 0);
        squares(head, c, a4, b4, sq, sk);
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) {
        part[0][threadIdx.x >> 5] = sq;
        part[1][threadIdx.x >> 5] = sk;
    }
    __syncthreads();
    const int n_warps = blockDim.x >> 5;
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
        sq += w < n_warps ? part[0][w] : 0.f;
        sk += w < n_warps ? part[1][w] : 0.f;
    }
    const float fq = qw ? rsqrtf(sq / (float)qc + eps) : 1.f, fk = kw ? rsqrtf(sk / (float)kc + eps) : 1.f;
    const long long at = at_s;

    auto finish = [&](int head, int c, const uint4& a4, const uint4& b4) {
        if (head < nh && head >= 0 ? false : at < 0) return;  // (no page: only the queries are written)
        if (head < 0) {
            const int g = c / e;
            *reinterpret_cast<uint4*>(v_pool + (at + (long long)g * page_size) * e + (c - g * e)) = a4;
            return;
        }
        const bool is_q = head < nh;
        const float f = is_q ? fq * (q_scale ? q_scale[head] : 1.f) : fk;
        const TW* w = is_q ? (qw ? qw + head * d + c : nullptr) : (kw ? kw + (head - nh) * d + c : nullptr);
        bf16* dst = (is_q ? xr + head * d : k_pool + (at + (long long)(head - nh) * page_size) * d) + c;
        float a[8], wv[8];
        unpack8(a4, a);
        if (w) load8(w, wv);
#pragma unroll
        for (int i = 0; i < 8; ++i) a[i] *= w ? f * wv[i] : f;
        if (c < half) {
            float b[8], sn[8], cs[8], ra[8], rb[8];
            unpack8(b4, b);
            if (w) load8(w + half, wv);
            load8(sn_s + c, sn);
            load8(cs_s + c, cs);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                b[i] *= w ? f * wv[i] : f;
                ra[i] = a[i] * cs[i] - b[i] * sn[i];
                rb[i] = b[i] * cs[i] + a[i] * sn[i];
            }
            *reinterpret_cast<uint4*>(dst) = pack8(ra);
            *reinterpret_cast<uint4*>(dst + half) = pack8(rb);
        } else {
            *reinterpret_cast<uint4*>(dst) = pack8(a);
        }
    };
#pragma unroll
    for (int n = 0; n < ROW_HOLD; ++n)
        if (threadIdx.x + n * blockDim.x < n_all) finish(head_of[n], c_of[n], ha[n], hb[n]);
    for (int it = threadIdx.x + ROW_HOLD * blockDim.x; it < n_all; it += blockDim.x) {
        int head, c;
        place(it, head, c);
        const bf16* src = xr + (head < 0 ? v_off : head * d) + c;
        finish(head, c, *reinterpret_cast<const uint4*>(src),
               head >= 0 && c < half ? *reinterpret_cast<const uint4*>(src + half) : make_uint4(0, 0, 0, 0));
    }
}

// x rows: [nh * d | nkv * d | ...], the values' nkv * e from column v_off on (behind the queries, which are written
// over; v_off = nh * d makes the keys, as they were projected, the values too); qw [nh * d] / kw [nkv * d] of type w_dtype (0 float32, 1 bf16), or
// null: not normed; q_scale float32 [nh] or null.
IB_EXPORT int ib_qk_row_norm_append(void* x, int x_stride, int dtype, const void* qw, const void* kw, int w_dtype, float eps,
                                    const float* q_scale, const float* inv_freq, int rd, const int* positions,
                                    const int* row_entry, const int* block_tables, int max_blocks, void* k_pool,
                                    void* v_pool, int n_rows, int nh, int nkv, int d, int e, int v_off, int page_size,
                                    int num_pages, unsigned* err, void* stream) {
    if (n_rows <= 0) return IB_OK;
    if (!x || !positions || !row_entry || !block_tables || !k_pool || !v_pool || !err) return IB_ERR_BAD_ARG;
    if (nh <= 0 || nkv <= 0 || d <= 0 || e <= 0 || page_size <= 0 || num_pages <= 0 || max_blocks <= 0 || rd < 0 ||
        (rd & 1) || rd > d || (rd > 0 && !inv_freq) || ((qw || kw) && !(eps > 0.f)) || w_dtype < 0 || w_dtype > 1)
        return IB_ERR_BAD_ARG;
    if (v_off < nh * d || x_stride < (nh + nkv) * d || x_stride < v_off + nkv * e) return IB_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t le;
#define IB_ROW(KERNEL, T, TW, THREADS)                                                                                   \
    le = launch_kernel(KERNEL, dim3(n_rows), dim3(THREADS), 0, s, (T*)x, x_stride, (const TW*)qw, (const TW*)kw, eps, q_scale, \
                       inv_freq, rd, positions, row_entry, block_tables, max_blocks, (T*)k_pool, (T*)v_pool, nh, nkv, d, e, v_off, \
                       page_size, num_pages, err)
    if (dtype == 1 && d % 8 == 0 && e % 8 == 0 && v_off % 8 == 0 && rd % 16 == 0 && rd / 2 <= ROW_MAX_PAIRS && x_stride % 8 == 0 &&
        !(((uintptr_t)x | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)qw | (uintptr_t)kw) & 15)) {
        const int items = (nh + nkv) * ((rd >> 4) + ((d - rd) >> 3)) + nkv * (e >> 3);
        const int threads = items <= 384 && n_rows >= 1024 ? 128 : 256;
        if (w_dtype == 0) IB_ROW(qk_row_norm_append_vec8_kernel<float>, bf16, float, threads);
        else IB_ROW(qk_row_norm_append_vec8_kernel<bf16>, bf16, bf16, threads);
    } else if (dtype == 0) {
        if (w_dtype == 0) IB_ROW((qk_row_norm_append_kernel<float, float>), float, float, 256);
        else IB_ROW((qk_row_norm_append_kernel<float, bf16>), float, bf16, 256);
    } else if (dtype == 1) {
        if (w_dtype == 0) IB_ROW((qk_row_norm_append_kernel<bf16, float>), bf16, float, 256);
        else IB_ROW((qk_row_norm_append_kernel<bf16, bf16>), bf16, bf16, 256);
    } else {
        return IB_ERR_UNSUPPORTED;
    }
#undef IB_ROW
    if (le != cudaSuccess) return (int)le;
    IB_LAUNCH_CHECK();
    return IB_OK;
}

template <typename T>
__global__ void attention_talk_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ k_pool,
                                      const T* __restrict__ v_pool, T* __restrict__ out, int out_stride,
                                      const float* __restrict__ talk, const T* __restrict__ gate, int gate_stride, const int* __restrict__ positions,
                                      const int* __restrict__ row_entry, const int* __restrict__ block_tables,
                                      int max_blocks, int nh, int nkv, int d, int e, int page_size, int num_pages,
                                      int chunk, int window, unsigned* __restrict__ err) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float sm[];
    constexpr int NK = 32, SS = NK + 1;
    float* qs = sm;                        // [nh][d]
    float* os = qs + nh * d;               // [nh][e]: running sums
    float* raw = os + nh * e;              // [nh][SS]
    float* mix = raw + nh * SS;            // [nh][SS]: combined scores, then weights
    float* mx = mix + nh * SS;             // [nh]
    float* den = mx + nh;                  // [nh]
    float* fac = den + nh;                 // [nh]
    __shared__ long long at_s[NK];         // each key's row among all rows of a pool (key/value head 0), or -1
    const int row = blockIdx.x, tid = threadIdx.x, R = nh / nkv;
    const int pos = positions[row];
    const int* table = block_tables + (size_t)row_entry[row] * max_blocks;
    for (int i = tid; i < nh * d; i += blockDim.x) qs[i] = to_f32(q[(size_t)row * q_stride + i]);
    for (int i = tid; i < nh * e; i += blockDim.x) os[i] = 0.f;
    for (int i = tid; i < nh; i += blockDim.x) {
        mx[i] = -INFINITY;
        den[i] = 0.f;
    }
    int lo = chunk > 0 ? pos / chunk * chunk : 0;
    if (window > 0) lo = max(lo, pos - window + 1);
    for (int j0 = lo / NK * NK; j0 <= pos; j0 += NK) {
        if (tid < NK) {
            const int j = j0 + tid;
            long long at = -1;
            if (j >= lo && j <= pos) {
                const int page = j / page_size < max_blocks ? table[j / page_size] : -1;
                if (page < 0 || page >= num_pages)
                    atomicOr(err, IB_FLAG_BAD_PAGE);
                else
                    at = (long long)page * nkv * page_size + j % page_size;
            }
            at_s[tid] = at;
        }
        __syncthreads();
        for (int i = tid; i < nh * NK; i += blockDim.x) {
            const int h = i / NK, t = i % NK;
            const long long at = at_s[t];
            float a = 0.f;
            if (at >= 0) {
                const T* kp = k_pool + (size_t)(at + (long long)(h / R) * page_size) * d;
                const float* qh = qs + h * d;
                for (int c = 0; c < d; ++c) a = fmaf(qh[c], to_f32(kp[c]), a);
            }
            raw[h * SS + t] = a;
        }
        __syncthreads();
        for (int i = tid; i < nh * NK; i += blockDim.x) {
            const int h = i / NK, t = i % NK;
            float a = -INFINITY;
            if (at_s[t] >= 0) {
                if (talk) {
                    a = 0.f;
                    for (int g = 0; g < nh; ++g) a = fmaf(talk[h * nh + g], raw[g * SS + t], a);
                } else {
                    a = raw[h * SS + t];
                }
            }
            mix[h * SS + t] = a;
        }
        __syncthreads();
        for (int h = tid >> 5; h < nh; h += blockDim.x >> 5) {
            const int t = tid & 31;
            const float s = mix[h * SS + t];
            const float n = fmaxf(mx[h], warp_max(s));
            const float p = s == -INFINITY ? 0.f : expf(s - n);
            const float sum = warp_sum(p);
            mix[h * SS + t] = p;
            __syncwarp();
            if (t == 0) {
                const float f = n == -INFINITY ? 1.f : expf(mx[h] - n);  // (exp(-inf) = 0 on the first keys)
                fac[h] = f;
                den[h] = den[h] * f + sum;
                mx[h] = n;
            }
        }
        __syncthreads();
        for (int i = tid; i < nh * e; i += blockDim.x) {
            const int h = i / e, c = i % e;
            float a = os[i] * fac[h];
            for (int t = 0; t < NK; ++t) {
                const long long at = at_s[t];
                if (at >= 0)
                    a = fmaf(mix[h * SS + t], to_f32(v_pool[(size_t)(at + (long long)(h / R) * page_size) * e + c]), a);
            }
            os[i] = a;
        }
        __syncthreads();
    }
    for (int i = tid; i < nh * e; i += blockDim.x) {
        const int h = i / e;
        float a = den[h] > 0.f ? os[i] / den[h] : 0.f;
        if (gate) a *= 1.f / (1.f + expf(-to_f32(gate[(size_t)row * gate_stride + h])));
        out[(size_t)row * out_stride + i] = from_f32<T>(a);
    }
}

// q rows of nh * d (stride q_stride), out rows of nh * e; talk float32 [nh, nh] or null (scores stay with their
// head), gate: one value of the activation dtype per (row, head) or null.
IB_EXPORT int ib_attention_talk(const void* q, int q_stride, const void* k_pool, const void* v_pool, void* out,
                                int out_stride, int dtype, const float* talk, const void* gate,
                                int gate_stride, const int* positions, const int* row_entry, const int* block_tables,
                                int max_blocks, int n_rows, int nh, int nkv, int d, int e, int page_size, int num_pages,
                                int chunk, int window, unsigned* err, void* stream) {
    if (n_rows <= 0) return IB_OK;
    if (!q || !k_pool || !v_pool || !out || !positions || !row_entry || !block_tables || !err) return IB_ERR_BAD_ARG;
    if (nh <= 0 || nkv <= 0 || nh % nkv || d <= 0 || e <= 0 || page_size <= 0 || num_pages <= 0 || max_blocks <= 0 ||
        q_stride < nh * d || out_stride < nh * e || (gate && gate_stride < nh) || chunk < 0 || window < 0)
        return IB_ERR_BAD_ARG;
    const size_t smem = ((size_t)nh * (d + e) + (size_t)nh * 2 * 33 + 3 * (size_t)nh) * sizeof(float);
    if (smem > 220 * 1024) return IB_ERR_TOO_LARGE;
    static bool configured = false;
    if (!configured) {
        cudaError_t ce = cudaFuncSetAttribute(attention_talk_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
        if (ce == cudaSuccess)
            ce = cudaFuncSetAttribute(attention_talk_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
        if (ce != cudaSuccess) return (int)ce;
        configured = true;
    }
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t le;
    if (dtype == 0)
        le = launch_kernel(attention_talk_kernel<float>, dim3(n_rows), dim3(256), smem, s, (const float*)q, q_stride,
                           (const float*)k_pool, (const float*)v_pool, (float*)out, out_stride, talk,
                           (const float*)gate, gate_stride, positions, row_entry, block_tables, max_blocks, nh, nkv, d, e,
                           page_size, num_pages, chunk, window, err);
    else if (dtype == 1)
        le = launch_kernel(attention_talk_kernel<bf16>, dim3(n_rows), dim3(256), smem, s, (const bf16*)q, q_stride,
                           (const bf16*)k_pool, (const bf16*)v_pool, (bf16*)out, out_stride, talk,
                           (const bf16*)gate, gate_stride, positions, row_entry, block_tables, max_blocks, nh, nkv, d, e,
                           page_size, num_pages, chunk, window, err);
    else
        return IB_ERR_UNSUPPORTED;
    if (le != cudaSuccess) return (int)le;
    IB_LAUNCH_CHECK();
    return IB_OK;
}

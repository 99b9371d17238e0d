// Attention whose heads exchange their scores before the softmax, on the tensor cores (bf16 mma.sync
// m16n8k16), for prompts and decoded tokens alike.  Compiled per (TALK_H, TALK_G, TALK_D, TALK_E): query
// heads, key/value heads, size of a key, size of a value.
//
//   r_g(i, j) = (q_g(i) . k_g(j)) * scale * temp_g        s_h(i, j) = sum_g talk[h, g] r_g(i, j)
//   out_h(i)  = sum_j softmax_j(s_h(i, .)) v_h(j) * sigmoid(gate_h(i))
//
// The exchange runs over all heads, so a CTA holds all heads of its eight queries: keys of every
// key/value head come in tiles of BN that start at absolute multiples of BN whatever the step's cut.
// A tile is worked on in three passes with a barrier between them:
//
//   1  a warp owns HW consecutive heads and computes S^T = K Q^T for each, [keys x 8 queries]; the
//      scaled scores go to shared memory as three bf16 numbers that add up to the 32-bit score (8
//      mantissa bits each), one plane a number, [query][key][head].
//   2  a warp takes a query: [heads x heads] (bf16, exact) times [heads x keys], the three planes one
//      after the other into one 32-bit accumulator: the exchange at 32-bit precision on the tensor
//      cores.  The result replaces the query's planes as 32-bit, [head][key].
//   3  a warp takes its heads again: running softmax over the tile and O^T += V^T P^T, [values x 8
//      queries] in registers.
//
// K has one stage (free after pass 1), V two; both of the next tile are fetched by cp.async during
// passes 2 and 3.  Key places are looked up in the block table once per tile, two tiles ahead.  Where
// all heads' accumulators do not fit the registers the values are cut in ES column blocks over CTAs,
// each of which computes the scores.
//
// Steps of few rows cut the keys in slices over CTAs; each writes its maxima, denominators and
// unnormed sums in 32-bit and a second kernel weighs them.
#include "common.cuh"

using namespace ib;

#ifndef TALK_H
#define TALK_H 32
#define TALK_G 8
#define TALK_D 128
#define TALK_E 128
#endif

namespace {
constexpr int H = TALK_H, G = TALK_G, D = TALK_D, E = TALK_E, R = H / G;
static_assert(H % G == 0 && D % 16 == 0 && E % 16 == 0 && D >= 16 && E >= 16, "sizes this kernel takes");
constexpr int gcd_of(int a, int b) { return b == 0 ? a : gcd_of(b, a % b); }
constexpr int BQ = 8;                               // queries of a CTA
constexpr int WARPS = H >= 8 ? 8 : 4, THREADS = WARPS * 32;
constexpr int HW = (H + WARPS - 1) / WARPS;         // heads of a warp
constexpr int SEG = gcd_of(HW, R);                  // of those, runs that share a key/value head
constexpr int HP = (H + 15) / 16 * 16;              // heads padded to the exchange's 16 x 16 pieces
constexpr int value_block() {
    for (int e = E; e >= 16; e -= 16)
        if (E % e == 0 && HW * e <= 512) return e;
    return 16;
}
constexpr int EB = value_block(), ES = E / EB;      // values in ES blocks of EB columns
constexpr int QS = D + 8, KS = D + 8, VS = EB + 8, SR = HP + 8;  // row strides (elements): 16 bytes of padding
constexpr int PLANES = 3;
constexpr bool alias_of(int bn) { return bn / 8 * (HP / 16) * 2 * PLANES <= 48; }
// Bytes of a query's region: the planes, and the exchanged scores in their place or behind them; the
// stride between queries is 8 words beyond a multiple of 32 banks.
constexpr int plane_bytes(int bn) { return bn * SR * 2; }
constexpr int mix_bytes(int bn) { return H * (bn + 8) * 4; }
constexpr int region_bytes(int bn) {
    int b = alias_of(bn) ? (PLANES * plane_bytes(bn) > mix_bytes(bn) ? PLANES * plane_bytes(bn) : mix_bytes(bn))
                         : PLANES * plane_bytes(bn) + mix_bytes(bn);
    b = (b + 127) / 128 * 128 + 32;
    return b;
}
constexpr int OUT_STAGE = WARPS * 8 * VS * 2;
constexpr int smem_bytes(int bn) {
    const int b = BQ * H * QS * 2 + G * bn * KS * 2 + 2 * G * bn * VS * 2 + BQ * region_bytes(bn) + HP * SR * 2 +
                  (H + 3) / 4 * 16 + 3 * bn * 4;
    return b > OUT_STAGE ? b : OUT_STAGE;
}
constexpr int SMEM_MAX = 227 * 1024;
constexpr int BN = smem_bytes(32) <= SMEM_MAX ? 32 : 16;  // keys of a tile
constexpr int SMEM = smem_bytes(BN);
constexpr bool FITS = SMEM <= SMEM_MAX && HW * EB <= 512;
constexpr bool ALIAS = alias_of(BN);
constexpr int QR = region_bytes(BN), PLANE = plane_bytes(BN), MIX_AT = ALIAS ? 0 : PLANES * PLANE, MS = BN + 8;
constexpr int MT = BN / 16, ET = EB / 16, KT = HP / 16;

__device__ __forceinline__ unsigned smem_addr(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm_x4(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldsm_x2(unsigned& r0, unsigned& r1, const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(r0), "=r"(r1) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldsm_x4_trans(unsigned& r0, unsigned& r1, unsigned& r2, unsigned& r3, const bf16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(smem_addr(p)));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const unsigned*>(&v);
}
__device__ __forceinline__ void cp_async16(bf16* smem, const bf16* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(smem_addr(smem)), "l"(gmem));
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;\n" ::: "memory"); }

struct Params {
    const bf16 *q, *k_pool, *v_pool, *gate;
    bf16* out;
    const float *talk, *temp;
    const int *cu_rows, *positions, *block_tables;
    int q_stride, out_stride, gate_stride, max_blocks, page_size, num_pages, chunk, window, splits, slice_len, n_rows;
    float scale;
    unsigned* err;
    float *stats, *part;  // [splits][rows][H][2], [splits][rows][H][E]
};

template <bool SPLIT>
__global__ void __launch_bounds__(THREADS, 1) attention_talk_mma_kernel(const Params p) {
    pdl_trigger();
    extern __shared__ __align__(128) unsigned char smem_raw[];
    bf16* qs = reinterpret_cast<bf16*>(smem_raw);          // [H][8][QS]
    bf16* ks = qs + H * BQ * QS;                           // [G][BN][KS]
    bf16* vs_all = ks + G * BN * KS;                       // [2][G][BN][VS]
    unsigned char* regions = reinterpret_cast<unsigned char*>(vs_all + 2 * G * BN * VS);  // [8][QR]
    bf16* ts = reinterpret_cast<bf16*>(regions + BQ * QR);  // [HP][SR]
    float* hs = reinterpret_cast<float*>(ts + HP * SR);     // [H] (padded to 4): scale * temperature
    int* places = reinterpret_cast<int*>(hs + (H + 3) / 4 * 4);  // [3][BN]: a key's row in the pool, -1: none

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    for (int i = tid; i < HP * HP; i += THREADS) {
        const int h = i / HP, g = i % HP;
        float v = 0.f;
        if (h < H && g < H) v = p.talk ? p.talk[h * H + g] : (h == g ? 1.f : 0.f);
        ts[h * SR + g] = __float2bfloat16_rn(v);
    }
    for (int i = tid; i < H; i += THREADS) hs[i] = p.scale * (p.temp ? p.temp[i] : 1.f);
    pdl_wait();

    const int en = blockIdx.y, sp = SPLIT ? blockIdx.z % p.splits : 0, eb = SPLIT ? blockIdx.z / p.splits : blockIdx.z;
    const int row0 = p.cu_rows[en], n_rows = p.cu_rows[en + 1] - row0;
    const int tile0 = (int)(gridDim.x - 1 - blockIdx.x) * BQ;  // (the last rows, which may see the most keys, first)
    if (tile0 >= n_rows) return;
    const int nq = min(BQ, n_rows - tile0);
    const int pos0 = p.positions[row0] + tile0, last = pos0 + nq - 1;  // an entry's rows are consecutive positions
    auto first_key = [&](int pos) {
        int lo = p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
        if (p.window > 0) lo = max(lo, pos - p.window + 1);
        return lo;
    };
    const int lo0 = first_key(pos0);
    int klo = lo0 / BN * BN, khi = last;
    if (SPLIT) {
        klo += sp * p.slice_len;
        khi = min(last, klo + p.slice_len - 1);
    }
    const int n_tiles = khi >= klo ? (khi - klo) / BN + 1 : 0;
    const int* table = p.block_tables + (size_t)en * p.max_blocks;
    const bf16* q_rows = p.q + (size_t)(row0 + tile0) * p.q_stride;

    auto look_up = [&](int t) {
        if (tid < BN) {
            const int j = klo + t * BN + tid;
            int at = -1;
            if (j >= lo0 && j <= khi) {
                const int page = j / p.page_size < p.max_blocks ? table[j / p.page_size] : -1;
                if (page < 0 || page >= p.num_pages)
                    atomicOr(p.err, IB_FLAG_BAD_PAGE);
                else
                    at = page * G * p.page_size + j % p.page_size;
            }
            places[t % 3 * BN + tid] = at;
        }
    };
    auto fetch = [&](int t) {
        const int* pl = places + t % 3 * BN;
        constexpr int KC = D / 8, VC = EB / 8;
        for (int c = tid; c < G * BN * KC; c += THREADS) {
            const int part = c % KC, key = c / KC % BN, g = c / (KC * BN), at = pl[key];
            bf16* dst = ks + (g * BN + key) * KS + part * 8;
            if (at >= 0)
                cp_async16(dst, p.k_pool + ((size_t)at + (size_t)g * p.page_size) * D + part * 8);
            else
                *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        bf16* vs = vs_all + (t & 1) * G * BN * VS;
        for (int c = tid; c < G * BN * VC; c += THREADS) {
            const int part = c % VC, key = c / VC % BN, g = c / (VC * BN), at = pl[key];
            bf16* dst = vs + (g * BN + key) * VS + part * 8;
            if (at >= 0)
                cp_async16(dst, p.v_pool + ((size_t)at + (size_t)g * p.page_size) * E + eb * EB + part * 8);
            else
                *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
    };

    {
        constexpr int QC = D / 8;
        for (int c = tid; c < BQ * H * QC; c += THREADS) {
            const int part = c % QC, h = c / QC % H, qi = c / (QC * H);
            bf16* dst = qs + (h * BQ + qi) * QS + part * 8;
            if (qi < nq)
                cp_async16(dst, q_rows + (size_t)qi * p.q_stride + h * D + part * 8);
            else
                *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
    }
    if (n_tiles > 0) {
        look_up(0);
        look_up(1);
        __syncthreads();
        fetch(0);
    }

    // this thread's query in pass 3 (a column of S^T and O^T is a query)
    const int my_pos = gq < nq ? pos0 + gq : -1, my_lo = gq < nq ? first_key(pos0 + gq) : 0;
    float o[HW][ET][4], mx[HW], den[HW];
#pragma unroll
    for (int a = 0; a < HW; ++a) {
        mx[a] = -INFINITY;
        den[a] = 0.f;
#pragma unroll
        for (int n = 0; n < ET; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) o[a][n][i] = 0.f;
    }

    for (int t = 0; t < n_tiles; ++t) {
        const int j0 = klo + t * BN;
        cp_async_wait_all();
        __syncthreads();
        // ---- pass 1: every head's scores
#pragma unroll
        for (int a = 0; a < HW; a += SEG) {
            const int h0 = warp * HW + a;
            if (h0 >= H) break;  // (the whole warp; a run of SEG heads exists or does not)
            const bf16* kg = ks + (h0 / R) * BN * KS + (lane & 15) * KS + (lane >> 4) * 8;
            float s[SEG][MT][4];
#pragma unroll
            for (int x = 0; x < SEG; ++x)
#pragma unroll
                for (int m = 0; m < MT; ++m)
#pragma unroll
                    for (int i = 0; i < 4; ++i) s[x][m][i] = 0.f;
#pragma unroll 4
            for (int kk = 0; kk < D / 16; ++kk) {
                unsigned ka[MT][4];
#pragma unroll
                for (int m = 0; m < MT; ++m) ldsm_x4(ka[m][0], ka[m][1], ka[m][2], ka[m][3], kg + m * 16 * KS + kk * 16);
                if (SEG % 2 == 0) {
#pragma unroll
                    for (int x = 0; x < SEG; x += 2) {
                        unsigned b0, b1, b2, b3;
                        ldsm_x4(b0, b1, b2, b3,
                                qs + ((h0 + x + (lane >> 4)) * BQ + (lane & 7)) * QS + kk * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
                        for (int m = 0; m < MT; ++m) {
                            mma_bf16(s[x][m], ka[m], b0, b1);
                            mma_bf16(s[x + (SEG > 1)][m], ka[m], b2, b3);
                        }
                    }
                } else {
#pragma unroll
                    for (int x = 0; x < SEG; ++x) {
                        unsigned b0, b1;
                        ldsm_x2(b0, b1, qs + ((h0 + x) * BQ + (lane & 7)) * QS + kk * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
                        for (int m = 0; m < MT; ++m) mma_bf16(s[x][m], ka[m], b0, b1);
                    }
                }
            }
            // scaled, in three bf16 numbers each (the differences are exact)
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int key = m * 16 + gq + (i >> 1) * 8, qi = 2 * tq + (i & 1);
                    bf16* dst = reinterpret_cast<bf16*>(regions + qi * QR) + key * SR + h0;
                    bf16 w[PLANES][SEG];
#pragma unroll
                    for (int x = 0; x < SEG; ++x) {
                        float v = s[x][m][i] * hs[h0 + x];
#pragma unroll
                        for (int l = 0; l < PLANES; ++l) {
                            w[l][x] = __float2bfloat16_rn(v);
                            v -= __bfloat162float(w[l][x]);
                        }
                    }
#pragma unroll
                    for (int l = 0; l < PLANES; ++l) {
                        bf16* d = dst + l * (PLANE / 2);
                        if (SEG % 4 == 0) {
#pragma unroll
                            for (int x = 0; x < SEG; x += 4) {
                                uint2 u;
                                u.x = (unsigned)__bfloat16_as_ushort(w[l][x]) |
                                      (unsigned)__bfloat16_as_ushort(w[l][x + (SEG > 1)]) << 16;
                                u.y = (unsigned)__bfloat16_as_ushort(w[l][x + 2 * (SEG > 2)]) |
                                      (unsigned)__bfloat16_as_ushort(w[l][x + 3 * (SEG > 3)]) << 16;
                                *reinterpret_cast<uint2*>(d + x) = u;
                            }
                        } else if (SEG % 2 == 0) {
#pragma unroll
                            for (int x = 0; x < SEG; x += 2)
                                *reinterpret_cast<unsigned*>(d + x) =
                                    (unsigned)__bfloat16_as_ushort(w[l][x]) |
                                    (unsigned)__bfloat16_as_ushort(w[l][x + (SEG > 1)]) << 16;
                        } else {
#pragma unroll
                            for (int x = 0; x < SEG; ++x) d[x] = w[l][x];
                        }
                    }
                }
        }
        if (HP != H) {  // heads that only fill up a piece: zeros, or what lies there would meet a zero weight
            constexpr int PADS = HP == H ? 1 : HP - H;
            for (int i = tid; i < BQ * BN * PADS; i += THREADS) {
                const int c = i % PADS, key = i / PADS % BN, qi = i / (PADS * BN);
                bf16* d = reinterpret_cast<bf16*>(regions + qi * QR) + key * SR + H + c;
#pragma unroll
                for (int l = 0; l < PLANES; ++l) d[l * (PLANE / 2)] = __float2bfloat16_rn(0.f);
            }
        }
        __syncthreads();
        if (t + 2 < n_tiles) look_up(t + 2);
        if (t + 1 < n_tiles) fetch(t + 1);
        // ---- pass 2: the exchange, a query at a time
        for (int qi = warp; qi < nq; qi += WARPS) {
            const bf16* raw = reinterpret_cast<const bf16*>(regions + qi * QR);
            float* mix = reinterpret_cast<float*>(regions + qi * QR + MIX_AT);
            constexpr int NT = BN / 8, GROUP = ALIAS ? NT : 2;  // tiles of 8 keys taken together
#pragma unroll
            for (int n0 = 0; n0 < NT; n0 += GROUP) {
                unsigned b[GROUP][KT][6];
#pragma unroll
                for (int n = 0; n < GROUP; ++n)
#pragma unroll
                    for (int kk = 0; kk < KT; ++kk) {
                        const bf16* src = raw + ((n0 + n) * 8 + (lane & 7)) * SR + kk * 16 + ((lane >> 3) & 1) * 8;
                        ldsm_x4(b[n][kk][0], b[n][kk][1], b[n][kk][2], b[n][kk][3], src + (lane >> 4) * (PLANE / 2));
                        ldsm_x2(b[n][kk][4], b[n][kk][5], src + 2 * (PLANE / 2));
                    }
                if (ALIAS) __syncwarp();  // (every lane has read before the planes are written over)
#pragma unroll
                for (int m = 0; m < KT; ++m) {
                    float c[GROUP][4];
#pragma unroll
                    for (int n = 0; n < GROUP; ++n)
#pragma unroll
                        for (int i = 0; i < 4; ++i) c[n][i] = 0.f;
#pragma unroll
                    for (int kk = 0; kk < KT; ++kk) {
                        unsigned a[4];
                        ldsm_x4(a[0], a[1], a[2], a[3], ts + (m * 16 + (lane & 15)) * SR + kk * 16 + (lane >> 4) * 8);
#pragma unroll
                        for (int l = PLANES - 1; l >= 0; --l)
#pragma unroll
                            for (int n = 0; n < GROUP; ++n) mma_bf16(c[n], a, b[n][kk][2 * l], b[n][kk][2 * l + 1]);
                    }
#pragma unroll
                    for (int n = 0; n < GROUP; ++n)
#pragma unroll
                        for (int i = 0; i < 2; ++i) {
                            const int h = m * 16 + gq + i * 8;
                            if (HP == H || h < H)
                                *reinterpret_cast<float2*>(mix + h * MS + (n0 + n) * 8 + 2 * tq) =
                                    make_float2(c[n][2 * i], c[n][2 * i + 1]);
                        }
                }
            }
        }
        __syncthreads();
        // ---- pass 3: softmax and values
        const bf16* vs = vs_all + (t & 1) * G * BN * VS;
        const float* mine = reinterpret_cast<const float*>(regions + gq * QR + MIX_AT);
#pragma unroll
        for (int a = 0; a < HW; a += SEG) {
            const int h0 = warp * HW + a;
            if (h0 >= H) break;
            unsigned pb[SEG][MT][2];
#pragma unroll
            for (int x = 0; x < SEG; ++x) {
                float s[MT][4], top = -INFINITY;
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    const float2 u = *reinterpret_cast<const float2*>(mine + (h0 + x) * MS + m * 16 + 2 * tq);
                    const float2 v = *reinterpret_cast<const float2*>(mine + (h0 + x) * MS + m * 16 + 2 * tq + 8);
                    s[m][0] = u.x;
                    s[m][1] = u.y;
                    s[m][2] = v.x;
                    s[m][3] = v.y;
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int j = j0 + m * 16 + 2 * tq + (i & 1) + (i >> 1) * 8;
                        if (j > my_pos || j < my_lo) s[m][i] = -INFINITY;
                        top = fmaxf(top, s[m][i]);
                    }
                }
                top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 1));
                top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 2));
                const float now = fmaxf(mx[a + x], top);
                const float f = now == mx[a + x] ? 1.f : __expf(mx[a + x] - now);  // (exp(-inf) = 0 on the first keys)
                mx[a + x] = now;
                float sum = 0.f;
#pragma unroll
                for (int m = 0; m < MT; ++m) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        s[m][i] = s[m][i] == -INFINITY ? 0.f : __expf(s[m][i] - now);
                        sum += s[m][i];
                    }
                    pb[x][m][0] = pack_bf16(s[m][0], s[m][1]);
                    pb[x][m][1] = pack_bf16(s[m][2], s[m][3]);
                }
                den[a + x] = den[a + x] * f + sum;  // (this thread's keys; added over the four at the end)
                if (__any_sync(0xffffffffu, f != 1.f)) {
                    const float f0 = __shfl_sync(0xffffffffu, f, 8 * tq), f1 = __shfl_sync(0xffffffffu, f, 8 * tq + 4);
#pragma unroll
                    for (int n = 0; n < ET; ++n) {
                        o[a + x][n][0] *= f0;
                        o[a + x][n][1] *= f1;
                        o[a + x][n][2] *= f0;
                        o[a + x][n][3] *= f1;
                    }
                }
            }
            const bf16* vg = vs + (h0 / R) * BN * VS + ((lane & 7) + (lane >> 4) * 8) * VS + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int n = 0; n < ET; ++n)
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    unsigned va[4];
                    ldsm_x4_trans(va[0], va[1], va[2], va[3], vg + m * 16 * VS + n * 16);
#pragma unroll
                    for (int x = 0; x < SEG; ++x) mma_bf16(o[a + x][n], va, pb[x][m][0], pb[x][m][1]);
                }
        }
    }

#pragma unroll
    for (int a = 0; a < HW; ++a) {
        den[a] += __shfl_xor_sync(0xffffffffu, den[a], 1);
        den[a] += __shfl_xor_sync(0xffffffffu, den[a], 2);
    }
    if (SPLIT) {
        cp_async_wait_all();  // (the queries, when the slice held no key)
#pragma unroll
        for (int a = 0; a < HW; ++a) {
            const int h = warp * HW + a;
            if (h >= H) break;
            const size_t base = (size_t)sp * p.n_rows + row0 + tile0;
            if (eb == 0 && tq == 0 && gq < nq) {
                float* st = p.stats + ((base + gq) * H + h) * 2;
                st[0] = mx[a];
                st[1] = den[a];
            }
            if (n_tiles == 0) continue;
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int qi = 2 * tq + i;
                if (qi >= nq) continue;
                float* dst = p.part + ((base + qi) * H + h) * E + eb * EB;
#pragma unroll
                for (int n = 0; n < ET; ++n) {
                    dst[n * 16 + gq] = o[a][n][i];
                    dst[n * 16 + gq + 8] = o[a][n][2 + i];
                }
            }
        }
        return;
    }
    // ---- gated, normed, through shared memory to rows of 16-byte stores
    __syncthreads();
    bf16* st = reinterpret_cast<bf16*>(smem_raw) + warp * 8 * VS;
#pragma unroll
    for (int a = 0; a < HW; ++a) {
        const int h = warp * HW + a;
        if (h >= H) break;
        float f = den[a] > 0.f ? 1.f / den[a] : 0.f;
        if (p.gate && gq < nq) {
            const float z = __bfloat162float(p.gate[(size_t)(row0 + tile0 + gq) * p.gate_stride + h]);
            f *= 1.f / (1.f + expf(-z));
        }
        const float f0 = __shfl_sync(0xffffffffu, f, 8 * tq), f1 = __shfl_sync(0xffffffffu, f, 8 * tq + 4);
#pragma unroll
        for (int n = 0; n < ET; ++n) {
            st[2 * tq * VS + n * 16 + gq] = __float2bfloat16_rn(o[a][n][0] * f0);
            st[(2 * tq + 1) * VS + n * 16 + gq] = __float2bfloat16_rn(o[a][n][1] * f1);
            st[2 * tq * VS + n * 16 + gq + 8] = __float2bfloat16_rn(o[a][n][2] * f0);
            st[(2 * tq + 1) * VS + n * 16 + gq + 8] = __float2bfloat16_rn(o[a][n][3] * f1);
        }
        __syncwarp();
        constexpr int OC = EB / 8;
        for (int c = lane; c < nq * OC; c += 32) {
            const int qi = c / OC, part = c % OC;
            *reinterpret_cast<uint4*>(p.out + (size_t)(row0 + tile0 + qi) * p.out_stride + h * E + eb * EB + part * 8) =
                *reinterpret_cast<const uint4*>(st + qi * VS + part * 8);
        }
        __syncwarp();
    }
}

// The slices weighed by their maxima, normed and gated: a CTA of four warps per (row, head); warp w adds the
// slices w, w + 4, ... and the four sums meet in shared memory in warp order.
__global__ void attention_talk_merge_kernel(const float* __restrict__ stats, const float* __restrict__ part,
                                            const bf16* __restrict__ gate, int gate_stride, bf16* __restrict__ out,
                                            int out_stride, int splits, int n_rows) {
    pdl_trigger();
    pdl_wait();
    __shared__ float sh_o[4][E];
    __shared__ float sh_l[4];
    const int item = blockIdx.x, row = item / H, h = item % H, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const size_t step = (size_t)n_rows * H;
    float best = -INFINITY;
    for (int k = lane; k < splits; k += 32) best = fmaxf(best, stats[(k * step + item) * 2]);
    best = warp_max(best);
    constexpr int PER = (E + 31) / 32;
    float o[PER], sum = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) o[i] = 0.f;
    for (int k = warp; k < splits; k += 4) {
        const float mk = stats[(k * step + item) * 2];
        if (mk == -INFINITY) continue;  // (the slice held no key of this row)
        const float f = expf(mk - best);
        sum = fmaf(stats[(k * step + item) * 2 + 1], f, sum);
        const float* src = part + (k * step + item) * E;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int c = lane + 32 * i;
            if (c < E) o[i] = fmaf(src[c], f, o[i]);
        }
    }
    if (lane == 0) sh_l[warp] = sum;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int c = lane + 32 * i;
        if (c < E) sh_o[warp][c] = o[i];
    }
    __syncthreads();
    const float l = ((sh_l[0] + sh_l[1]) + sh_l[2]) + sh_l[3];
    float f = l > 0.f ? 1.f / l : 0.f;
    if (gate) f *= 1.f / (1.f + expf(-__bfloat162float(gate[(size_t)row * gate_stride + h])));
    for (int c = threadIdx.x; c < E; c += 128)
        out[(size_t)row * out_stride + h * E + c] =
            __float2bfloat16_rn((((sh_o[0][c] + sh_o[1][c]) + sh_o[2][c]) + sh_o[3][c]) * f);
}
}  // namespace

// What was compiled: sizes, keys of a tile, blocks of the values, whether the shared memory suffices.
IB_EXPORT int ib_attention_talk_mma_info(int what) {
    const int v[] = {H, G, D, E, BN, ES, FITS ? 1 : 0, SMEM};
    return what >= 0 && what < 8 ? v[what] : -1;
}

IB_EXPORT long long ib_attention_talk_mma_scratch_bytes(int n_rows, int splits) {
    return (long long)splits * n_rows * H * (2 + E) * (long long)sizeof(float);
}

// q rows begin with H * D queries (row stride q_stride), out rows hold H * E (stride out_stride); talk float32 [H, H]
// whose values are exact in bf16, or null; temp float32 [H] or null; gate bf16, one per (row, head), or null.
// max_rows: an upper bound on the rows of any entry (the grid's width).  splits > 1: the keys from the first
// that a CTA's first query sees, rounded down to the key tile, in slices of `slice_len` (a multiple of the key
// tile; together they must reach the last query) over that many CTAs, through `scratch`; n_rows: all rows.
IB_EXPORT int ib_attention_talk_mma(const void* q, int q_stride, const void* k_pool, const void* v_pool, void* out,
                                    int out_stride, const float* talk, const float* temp, const void* gate,
                                    int gate_stride, const int* cu_rows, const int* positions, const int* block_tables,
                                    int max_blocks, int n_entries, int max_rows, int page_size, int num_pages,
                                    float scale, int chunk, int window, unsigned* err, int n_rows, int splits,
                                    int slice_len, void* scratch, long long scratch_bytes, void* stream) {
    if (n_entries <= 0 || max_rows <= 0 || n_rows <= 0) return IB_OK;
    if (!q || !k_pool || !v_pool || !out || !cu_rows || !positions || !block_tables || !err) return IB_ERR_BAD_ARG;
    if (page_size <= 0 || num_pages <= 0 || max_blocks <= 0 || chunk < 0 || window < 0 || splits < 1 ||
        q_stride < H * D || out_stride < H * E || (gate && gate_stride < H))
        return IB_ERR_BAD_ARG;
    if (!FITS || q_stride % 8 || out_stride % 8 || (((uintptr_t)q | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)out) & 15))
        return IB_ERR_UNSUPPORTED;
    if (n_entries > 65535 || (long long)splits * ES > 65535 || (long long)num_pages * G * page_size > 0x7fffffffLL)
        return IB_ERR_TOO_LARGE;
    static bool configured = false;
    if (!configured) {
        cudaError_t ce = cudaFuncSetAttribute(attention_talk_mma_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
        if (ce == cudaSuccess)
            ce = cudaFuncSetAttribute(attention_talk_mma_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
        if (ce != cudaSuccess) return (int)ce;
        configured = true;
    }
    Params p;
    p.q = (const bf16*)q;
    p.k_pool = (const bf16*)k_pool;
    p.v_pool = (const bf16*)v_pool;
    p.gate = (const bf16*)gate;
    p.out = (bf16*)out;
    p.talk = talk;
    p.temp = temp;
    p.cu_rows = cu_rows;
    p.positions = positions;
    p.block_tables = block_tables;
    p.q_stride = q_stride;
    p.out_stride = out_stride;
    p.gate_stride = gate_stride;
    p.max_blocks = max_blocks;
    p.page_size = page_size;
    p.num_pages = num_pages;
    p.chunk = chunk;
    p.window = window;
    p.splits = splits;
    p.slice_len = slice_len;
    p.n_rows = n_rows;
    p.scale = scale;
    p.err = err;
    p.stats = nullptr;
    p.part = nullptr;
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 grid((max_rows + BQ - 1) / BQ, n_entries, ES * splits);
    cudaError_t le;
    if (splits == 1) {
        le = launch_kernel(attention_talk_mma_kernel<false>, grid, dim3(THREADS), SMEM, s, p);
        if (le != cudaSuccess) return (int)le;
        IB_LAUNCH_CHECK();
        return IB_OK;
    }
    if (!scratch || slice_len <= 0 || slice_len % BN || scratch_bytes < ib_attention_talk_mma_scratch_bytes(n_rows, splits))
        return IB_ERR_BAD_ARG;
    p.stats = (float*)scratch;
    p.part = p.stats + (size_t)splits * n_rows * H * 2;
    le = launch_kernel(attention_talk_mma_kernel<true>, grid, dim3(THREADS), SMEM, s, p);
    if (le != cudaSuccess) return (int)le;
    le = launch_kernel(attention_talk_merge_kernel, dim3((unsigned)((long long)n_rows * H)), dim3(128), 0, s,
                       (const float*)p.stats, (const float*)p.part, p.gate, gate_stride, p.out, out_stride, splits, n_rows);
    if (le != cudaSuccess) return (int)le;
    IB_LAUNCH_CHECK();
    return IB_OK;
}

// Attention whose heads exchange their scores before the softmax, on the tensor cores (bf16 mma.sync
// m16n8k16), for prompts and decoded tokens alike.  Compiled per (TALK_H, TALK_G, TALK_D, TALK_E): query
// heads, key/value heads, size of a key, size of a value.
//
//   s_h(i, j) = sum_g talk[h, g] (q_g(i) . k_g(j))
//   out_h(i)  = sum_j softmax_j(s_h(i, .)) v_h(j) * sigmoid(gate_h(i))
//
// (scales of the scores are in the queries, which qk_row_norm_append scales before it rounds them).
//
// The exchange runs over all heads, so a CTA holds all heads of its BQ queries (8; for decoded tokens as
// many as fill eight columns of one key/value head): keys of every key/value head come in tiles of BN that
// start at absolute multiples of BN whatever the step's cut.  The columns of a key/value head are its
// (query, head) pairs, query by query; a unit is eight of them, and a warp owns UW units.  A tile is
// worked on in three passes:
//
//   1  S^T = K Q^T per unit, [keys x 8 columns]; the scores go to shared memory as three bf16
//      numbers that add up to the 32-bit score (8 mantissa bits each), one plane a number,
//      [query][key][head].
//   2  per query, 16 heads and 16 keys: [heads x heads] (bf16, exact) times [heads x keys], the three
//      planes one after the other into one 32-bit accumulator: the exchange at 32-bit precision on the
//      tensor cores.  The result goes to shared memory as 32-bit, [query][head][key].
//   3  per unit: running softmax over the tile and O^T += V^T P^T, [values x 8 columns] in registers.
//
// For prompts pass 3 of a tile and pass 1 of the next share the stretch between two barriers; keys have two
// stages then (where they fit), values one, fetched by cp.async during pass 2.  Otherwise keys have one
// stage, fetched while passes 2 and 3 of the tile before run, and values one, fetched during passes 1 and
// 2, which leaves room for a second CTA on the SM.  Key places are looked up in the block table once per tile, two
// tiles ahead.  Where the accumulators do not fit the registers the values are cut in ES column blocks
// over CTAs, each of which computes the scores.
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
constexpr int HP = (H + 15) / 16 * 16;              // heads padded to the exchange's 16 x 16 pieces
constexpr int KT = HP / 16;
constexpr int SR = HP + 8, QS = D + 8, KS = D + 8;  // row strides (elements): 16 bytes of padding
constexpr int PLANES = 3;
constexpr int SMEM_MAX = 227 * 1024;
constexpr int BQ_FEW = R >= 8 ? 1 : 8 / R;          // queries of a CTA when every entry has few rows

template <int BQ>
struct Cfg {
    static constexpr int UPG = (BQ * R + 7) / 8;    // units of a key/value head
    static constexpr int NU = G * UPG;
    static constexpr int WARPS = NU >= 16 && BQ == 8 ? 16 : (NU >= 8 ? 8 : 4);
    static constexpr int THREADS = WARPS * 32;
    static constexpr int UW = (NU + WARPS - 1) / WARPS;
    static constexpr int SEG = gcd_of(UW, UPG);     // of a warp's units, runs that share a key/value head
    static constexpr int MOST = WARPS == 16 ? 256 : 512;  // UW * EB: accumulators that fit the registers
    static constexpr int value_block() {
        for (int e = E; e >= 16; e -= 16)
            if (E % e == 0 && UW * e <= MOST) return e;
        return 16;
    }
    static constexpr int EB = value_block(), ES = E / EB;  // values in ES blocks of EB columns
    static constexpr int VS = EB + 8, ET = EB / 16;
    static constexpr int plane_bytes(int bn) { return bn * SR * 2; }
    // A query's region: the planes, then the exchanged scores; 8 words beyond a multiple of the 32 banks.
    static constexpr int region_bytes(int bn) { return (PLANES * plane_bytes(bn) + H * (bn + 8) * 4 + 127) / 128 * 128 + 32; }
    static constexpr int smem_bytes(int bn, int stages = 1) {
        const int b = G * UPG * 8 * QS * 2 + stages * G * bn * KS * 2 + G * bn * VS * 2 + BQ * region_bytes(bn) + HP * SR * 2 +
                      3 * bn * 4;
        const int st = WARPS * 8 * VS * 2;
        return b > st ? b : st;
    }
    // keys of a tile: for few rows as many as leave room for a second CTA on the SM, if any do
    static constexpr int pick() {
        if (BQ != 8 || BQ_FEW == 8) {
            if (smem_bytes(32) <= SMEM_MAX / 2 - 1024) return 32;
            if (smem_bytes(16) <= SMEM_MAX / 2 - 1024) return 16;
        }
        return smem_bytes(32) <= SMEM_MAX ? 32 : 16;
    }
    static constexpr int BN = pick(), KST = BQ == 8 && smem_bytes(BN, 2) <= SMEM_MAX ? 2 : 1, SMEM = smem_bytes(BN, KST), QR = region_bytes(BN), PLANE = plane_bytes(BN),
                         MIX_AT = PLANES * PLANE, MS = BN + 8, MT = BN / 16;
    static constexpr bool FITS = SMEM <= SMEM_MAX && UW * EB <= MOST;
};

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
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_but_one() { asm volatile("cp.async.wait_group 1;\n" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;\n" ::: "memory"); }

template <int N>
struct Int {
    static constexpr int value = N;
};
// 2^x by the special function unit, results below the normal range as zero; log2(e)
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
    return y;
}
constexpr float LOG2E = 1.4426950408889634f;

struct Params {
    const bf16 *q, *k_pool, *v_pool, *gate;
    bf16* out;
    const float* talk;
    const int *cu_rows, *positions, *block_tables;
    int q_stride, out_stride, gate_stride, max_blocks, page_size, num_pages, chunk, window, splits, slice_len, n_rows, run_tiles;
    unsigned* err;
    float *stats, *part;  // [splits][rows][H][2] (maxima times log2(e)), [splits][rows][H][E]
};

template <int BQ, bool SPLIT>
__global__ void __launch_bounds__(Cfg<BQ>::THREADS, 1) attention_talk_mma_kernel(const Params p) {
    using C = Cfg<BQ>;
    constexpr int UPG = C::UPG, NU = C::NU, WARPS = C::WARPS, THREADS = C::THREADS, UW = C::UW, SEG = C::SEG, EB = C::EB,
                  VS = C::VS, ET = C::ET, BN = C::BN, QR = C::QR, PLANE = C::PLANE, MIX_AT = C::MIX_AT, MS = C::MS,
                  MT = C::MT;
    pdl_trigger();
    extern __shared__ __align__(128) unsigned char smem_raw[];
    bf16* qs = reinterpret_cast<bf16*>(smem_raw);            // [NU * 8 columns][QS]
    bf16* ks = qs + NU * 8 * QS;                             // [KST][G][BN][KS]
    bf16* vs = ks + C::KST * G * BN * KS;                           // [G][BN][VS]
    unsigned char* regions = reinterpret_cast<unsigned char*>(vs + G * BN * VS);  // [BQ][QR]
    bf16* ts = reinterpret_cast<bf16*>(regions + BQ * QR);   // [HP][SR]
    int* places = reinterpret_cast<int*>(ts + HP * SR);      // [3][BN]: a key's row in the pool, -1: none

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    for (int i = tid; i < HP * HP; i += THREADS) {
        const int h = i / HP, g = i % HP;
        float v = 0.f;
        if (h < H && g < H) v = p.talk ? p.talk[h * H + g] : (h == g ? 1.f : 0.f);
        ts[h * SR + g] = __float2bfloat16_rn(v);
    }
    if (HP != H) {  // heads that only fill up a piece: zeros, or what lies there would meet a zero weight
        constexpr int PADS = HP == H ? 1 : HP - H;
        for (int i = tid; i < BQ * PLANES * BN * PADS; i += THREADS) {
            const int c = i % PADS, key = i / PADS % (PLANES * BN), qi = i / (PADS * PLANES * BN);
            reinterpret_cast<bf16*>(regions + qi * QR)[key * SR + H + c] = __float2bfloat16_rn(0.f);
        }
    }
    pdl_wait();

    const int en = blockIdx.y, sp = SPLIT ? blockIdx.z % p.splits : 0, eb = SPLIT ? blockIdx.z / p.splits : blockIdx.z;
    const int row0 = p.cu_rows[en], n_rows = p.cu_rows[en + 1] - row0;
    // The rows that see the most keys first: the last ones or, with several runs of positions in an entry, the
    // last of every run, then those before them.
    int tile = (int)(gridDim.x - 1 - blockIdx.x);
    if (p.run_tiles > 0) {
        const int runs = (int)gridDim.x / p.run_tiles;
        tile = (int)blockIdx.x % runs * p.run_tiles + p.run_tiles - 1 - (int)blockIdx.x / runs;
    }
    const int tile0 = tile * BQ;
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
    // rows of W elements of all key/value heads, 16 bytes a copy; where the threads cover whole tiles of one
    // key/value head a thread's key stays the same from one to the next
    auto fetch_rows = [&](bf16* dst, int dst_stride, const bf16* pool, int pool_width, auto width, const int* pl) {
        constexpr int PARTS = decltype(width)::value / 8, HEAD = BN * PARTS;
        const size_t head_step = (size_t)p.page_size * pool_width;
        if constexpr (THREADS % HEAD == 0) {
            const int part = tid % PARTS, key = tid / PARTS % BN, at = pl[key];
            bf16* d = dst + (tid / HEAD * BN + key) * dst_stride + part * 8;
            const bf16* src = pool + (size_t)(at < 0 ? 0 : at) * pool_width + part * 8 + tid / HEAD * head_step;
#pragma unroll
            for (int g = 0; g < G; g += THREADS / HEAD) {
                if (G % (THREADS / HEAD) != 0 && g + tid / HEAD >= G) break;
                if (at >= 0) cp_async16(d, src);
                else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
                d += THREADS / HEAD * BN * dst_stride;
                src += THREADS / HEAD * head_step;
            }
        } else {
            for (int c = tid; c < G * HEAD; c += THREADS) {
                const int part = c % PARTS, key = c / PARTS % BN, g = c / HEAD, at = pl[key];
                bf16* d = dst + (g * BN + key) * dst_stride + part * 8;
                if (at >= 0) cp_async16(d, pool + (size_t)at * pool_width + g * head_step + part * 8);
                else *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
            }
        }
        cp_async_commit();
    };
    auto fetch_keys = [&](int t) { fetch_rows(ks + t % C::KST * G * BN * KS, KS, p.k_pool, D, Int<D>{}, places + t % 3 * BN); };
    auto fetch_values = [&](int t) { fetch_rows(vs, VS, p.v_pool + eb * EB, E, Int<EB>{}, places + t % 3 * BN); };

    {
        constexpr int QC = D / 8;
        for (int c = tid; c < NU * 8 * QC; c += THREADS) {
            const int part = c % QC, col = c / QC % (UPG * 8), g = c / (QC * UPG * 8), qi = col / R;
            bf16* dst = qs + (g * UPG * 8 + col) * QS + part * 8;
            if (qi < nq)
                cp_async16(dst, q_rows + (size_t)qi * p.q_stride + (g * R + col % R) * D + part * 8);
            else
                *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        cp_async_commit();
    }
    if (n_tiles > 0) {
        look_up(0);
        look_up(1);
        __syncthreads();
        fetch_keys(0);
    }

    // Per unit: where this thread's two columns of S^T (pass 1) go, what its one column of P^T (pass 3: column gq)
    // reads and sees.  Columns that only fill up a unit, and queries beyond the entry's last, write nowhere
    // and see nothing.
    int raw_a[UW], raw_b[UW], mix_at[UW], sees_lo[UW], sees_hi[UW];
#pragma unroll
    for (int a = 0; a < UW; ++a) {
        const int u = warp * UW + a, g = u / UPG, c0 = u % UPG * 8 + 2 * tq, c = u % UPG * 8 + gq;
        raw_a[a] = c0 < BQ * R ? c0 / R * QR + gq * SR * 2 + (g * R + c0 % R) * 2 : -1;
        raw_b[a] = c0 + 1 < BQ * R ? (c0 + 1) / R * QR + gq * SR * 2 + (g * R + (c0 + 1) % R) * 2 : -1;
        const bool live = u < NU && c / R < nq;
        mix_at[a] = (live ? c / R * QR + (g * R + c % R) * MS * 4 : 0) + MIX_AT + 8 * tq;
        sees_hi[a] = live ? pos0 + c / R - 2 * tq : -1 - 2 * tq;
        sees_lo[a] = live ? first_key(pos0 + c / R) - 2 * tq : 0;
    }
    const int lo_last = first_key(last);
    // mx: running maximum, in units of log2(e)
    float o[UW][ET][4], mx[UW], den[UW];
#pragma unroll
    for (int a = 0; a < UW; ++a) {
        mx[a] = -INFINITY;
        den[a] = 0.f;
#pragma unroll
        for (int n = 0; n < ET; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) o[a][n][i] = 0.f;
    }

    // ---- pass 1: the scores of every unit
    auto pass1 = [&](const bf16* ks_now) {
#pragma unroll
        for (int a = 0; a < UW; a += SEG) {
            const int u0 = warp * UW + a;
            if (u0 >= NU) break;  // (the whole warp; a run of SEG units exists or does not)
            const int g = u0 / UPG;
            const bf16* kg = ks_now + g * BN * KS + (lane & 15) * KS + (lane >> 4) * 8;
            const bf16* qu = qs + (u0 * 8 + (lane & 7)) * QS;
            float s[SEG][MT][4];
#pragma unroll
            for (int x = 0; x < SEG; ++x)
#pragma unroll
                for (int m = 0; m < MT; ++m)
#pragma unroll
                    for (int i = 0; i < 4; ++i) s[x][m][i] = 0.f;
            // two steps of 16 at a time: one load of a unit's columns serves both
#pragma unroll 2
            for (int kk = 0; kk + 2 <= D / 16; kk += 2) {
                unsigned ka[2][MT][4], b[SEG][4];
#pragma unroll
                for (int m = 0; m < MT; ++m)
#pragma unroll
                    for (int y = 0; y < 2; ++y)
                        ldsm_x4(ka[y][m][0], ka[y][m][1], ka[y][m][2], ka[y][m][3], kg + m * 16 * KS + (kk + y) * 16);
#pragma unroll
                for (int x = 0; x < SEG; ++x)
                    ldsm_x4(b[x][0], b[x][1], b[x][2], b[x][3], qu + x * 8 * QS + kk * 16 + (lane >> 3) * 8);
#pragma unroll
                for (int y = 0; y < 2; ++y)
#pragma unroll
                    for (int x = 0; x < SEG; ++x)
#pragma unroll
                        for (int m = 0; m < MT; ++m) mma_bf16(s[x][m], ka[y][m], b[x][2 * y], b[x][2 * y + 1]);
            }
            if (D / 16 % 2) {
                constexpr int kk = D / 16 - 1;
                unsigned ka[4];
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    ldsm_x4(ka[0], ka[1], ka[2], ka[3], kg + m * 16 * KS + kk * 16);
#pragma unroll
                    for (int x = 0; x < SEG; ++x) {
                        unsigned b0, b1;
                        ldsm_x2(b0, b1, qu + x * 8 * QS + kk * 16 + ((lane >> 3) & 1) * 8);
                        mma_bf16(s[x][m], ka, b0, b1);
                    }
                }
            }
            // in three bf16 numbers each: the leading bits, twice, and the rest (the differences are exact)
#pragma unroll
            for (int x = 0; x < SEG; ++x)
#pragma unroll
                for (int m = 0; m < MT; ++m)
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        float va = s[x][m][2 * i], vb = s[x][m][2 * i + 1];
                        const int at = (m * 16 + i * 8) * SR * 2;
#pragma unroll
                        for (int l = 0; l < PLANES; ++l) {
                            const unsigned ia = __float_as_uint(va), ib = __float_as_uint(vb);
                            const unsigned w = __byte_perm(ia, ib, 0x7632);  // both upper halves
                            if (l + 1 < PLANES) {
                                va -= __uint_as_float(ia & 0xffff0000u);
                                vb -= __uint_as_float(ib & 0xffff0000u);
                            }
                            unsigned char* d = regions + at + l * PLANE;
                            if (R % 2 == 0) {
                                if (BQ * R % 8 == 0 || raw_a[a + x] >= 0) *reinterpret_cast<unsigned*>(d + raw_a[a + x]) = w;
                            } else {
                                if (BQ * R % 8 == 0 || raw_a[a + x] >= 0)
                                    *reinterpret_cast<unsigned short*>(d + raw_a[a + x]) = (unsigned short)w;
                                if (BQ * R % 8 == 0 || raw_b[a + x] >= 0)
                                    *reinterpret_cast<unsigned short*>(d + raw_b[a + x]) = (unsigned short)(w >> 16);
                            }
                        }
                    }
        }
    };
    // ---- pass 2: the exchange; an item is a query, 16 heads and 16 keys
    auto pass2 = [&]() {
        for (int it = warp; it < nq * KT * MT; it += WARPS) {
            const int n0 = it % MT * 2, m = it / MT % KT, qi = it / (MT * KT);
            const bf16* raw = reinterpret_cast<const bf16*>(regions + qi * QR) + (n0 * 8 + (lane & 7)) * SR + ((lane >> 3) & 1) * 8;
            float* mix = reinterpret_cast<float*>(regions + qi * QR + MIX_AT);
            float c[2][4];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int i = 0; i < 4; ++i) c[n][i] = 0.f;
#pragma unroll 2
            for (int kk = 0; kk < KT; ++kk) {
                unsigned a[4], b[PLANES][4];
                ldsm_x4(a[0], a[1], a[2], a[3], ts + (m * 16 + (lane & 15)) * SR + kk * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int l = 0; l < PLANES; ++l)  // both tiles of 8 keys
                    ldsm_x4(b[l][0], b[l][1], b[l][2], b[l][3], raw + (lane >> 4) * 8 * SR + kk * 16 + l * (PLANE / 2));
#pragma unroll
                for (int l = PLANES - 1; l >= 0; --l)
#pragma unroll
                    for (int n = 0; n < 2; ++n) mma_bf16(c[n], a, b[l][2 * n], b[l][2 * n + 1]);
            }
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int h = m * 16 + gq + i * 8;
                    if (HP == H || h < H)
                        *reinterpret_cast<float2*>(mix + h * MS + (n0 + n) * 8 + 2 * tq) = make_float2(c[n][2 * i], c[n][2 * i + 1]);
                }
        }
    };
    // ---- pass 3: softmax and values
    auto pass3 = [&](int j0) {
        const bool all_seen = nq == BQ && j0 >= lo_last && j0 + BN - 1 <= pos0;
#pragma unroll
        for (int a = 0; a < UW; a += SEG) {
            const int u0 = warp * UW + a;
            if (u0 >= NU) break;
            const int g = u0 / UPG;
            unsigned pb[SEG][MT][2];
#pragma unroll
            for (int x = 0; x < SEG; ++x) {
                const float* mine = reinterpret_cast<const float*>(regions + mix_at[a + x]);
                float s[MT][4], top = -INFINITY;
#pragma unroll
                for (int m = 0; m < MT; ++m) {
                    const float2 u = *reinterpret_cast<const float2*>(mine + m * 16);
                    const float2 v = *reinterpret_cast<const float2*>(mine + m * 16 + 8);
                    s[m][0] = u.x;
                    s[m][1] = u.y;
                    s[m][2] = v.x;
                    s[m][3] = v.y;
                }
                if (!all_seen) {
#pragma unroll
                    for (int m = 0; m < MT; ++m)
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            const int j = j0 + m * 16 + (i & 1) + (i >> 1) * 8;
                            if (j > sees_hi[a + x] || j < sees_lo[a + x]) s[m][i] = -INFINITY;
                        }
                }
#pragma unroll
                for (int m = 0; m < MT; ++m)
#pragma unroll
                    for (int i = 0; i < 4; ++i) top = fmaxf(top, s[m][i]);
                top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 1));
                top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 2));
                const float now = fmaxf(mx[a + x], top * LOG2E);
                const float f = now == mx[a + x] ? 1.f : exp2_fast(mx[a + x] - now);  // (2^-inf = 0 on the first keys)
                const float from = now == -INFINITY ? 0.f : now;
                mx[a + x] = now;
                float sum = 0.f;
#pragma unroll
                for (int m = 0; m < MT; ++m) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        s[m][i] = exp2_fast(fmaf(s[m][i], LOG2E, -from));  // (2^-inf = 0 for keys that are not seen)
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
            const bf16* vg = vs + g * BN * VS + ((lane & 7) + (lane >> 4) * 8) * VS + ((lane >> 3) & 1) * 8;
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
    };

    if constexpr (C::KST == 2) {
        // Two barriers a tile: between one and the next the exchange of tile t, then softmax and values of tile t
        // beside the scores of tile t + 1, which need nothing of one another.
        if (n_tiles > 0) {
            cp_async_wait_all();
            __syncthreads();
            if (n_tiles > 1) fetch_keys(1);
            pass1(ks);
        }
        for (int t = 0; t < n_tiles; ++t) {
            __syncthreads();
            fetch_values(t);
            if (t + 2 < n_tiles) look_up(t + 2);
            pass2();
            cp_async_wait_all();  // the values of tile t and the keys of tile t + 1
            __syncthreads();
            if (t + 2 < n_tiles) fetch_keys(t + 2);
            pass3(klo + t * BN);
            if (t + 1 < n_tiles) pass1(ks + ((t + 1) & 1) * G * BN * KS);
        }
    } else {
        for (int t = 0; t < n_tiles; ++t) {
            cp_async_wait_all();
            __syncthreads();
            fetch_values(t);
            pass1(ks);
            __syncthreads();
            if (t + 2 < n_tiles) look_up(t + 2);
            if (t + 1 < n_tiles) fetch_keys(t + 1);
            pass2();
            if (t + 1 < n_tiles) cp_async_wait_but_one();  // the values are here; the next keys need not be
            else cp_async_wait_all();
            __syncthreads();
            pass3(klo + t * BN);
        }
    }

#pragma unroll
    for (int a = 0; a < UW; ++a) {
        den[a] += __shfl_xor_sync(0xffffffffu, den[a], 1);
        den[a] += __shfl_xor_sync(0xffffffffu, den[a], 2);
    }
    if (SPLIT) {
        cp_async_wait_all();  // (the queries, when the slice held no key)
#pragma unroll
        for (int a = 0; a < UW; ++a) {
            const int u = warp * UW + a;
            if (u >= NU) break;
            const int g = u / UPG, c0 = u % UPG * 8;
            const size_t base = (size_t)sp * p.n_rows + row0 + tile0;
            if (eb == 0 && tq == 0 && (c0 + gq) / R < nq) {
                float* st = p.stats + ((base + (c0 + gq) / R) * H + g * R + (c0 + gq) % R) * 2;
                st[0] = mx[a];
                st[1] = den[a];
            }
            if (n_tiles == 0) continue;
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int c = c0 + 2 * tq + i;
                if (c / R >= nq) continue;
                float* dst = p.part + ((base + c / R) * H + g * R + c % R) * E + eb * EB;
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
    for (int a = 0; a < UW; ++a) {
        const int u = warp * UW + a;
        if (u >= NU) break;
        const int g = u / UPG, c0 = u % UPG * 8;
        float f = den[a] > 0.f ? 1.f / den[a] : 0.f;
        if (p.gate && (c0 + gq) / R < nq) {
            const float z = __bfloat162float(p.gate[(size_t)(row0 + tile0 + (c0 + gq) / R) * p.gate_stride + g * R + (c0 + gq) % R]);
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
        for (int x = lane; x < 8 * OC; x += 32) {
            const int col = x / OC, part = x % OC, qi = (c0 + col) / R;
            if (qi < nq)
                *reinterpret_cast<uint4*>(p.out + (size_t)(row0 + tile0 + qi) * p.out_stride + (g * R + (c0 + col) % R) * E +
                                          eb * EB + part * 8) = *reinterpret_cast<const uint4*>(st + col * VS + part * 8);
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
        const float f = exp2_fast(mk - best);
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

template <int BQ>
int launch_talk(const Params& p, int n_entries, int max_rows, cudaStream_t s) {
    using C = Cfg<BQ>;
    if (!C::FITS) return IB_ERR_UNSUPPORTED;
    if ((long long)p.splits * C::ES > 65535) return IB_ERR_TOO_LARGE;
    if (p.splits > 1 && (p.slice_len <= 0 || p.slice_len % C::BN)) return IB_ERR_BAD_ARG;
    static bool configured = false;
    if (!configured) {
        cudaError_t ce = cudaFuncSetAttribute(attention_talk_mma_kernel<BQ, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM);
        if (ce == cudaSuccess)
            ce = cudaFuncSetAttribute(attention_talk_mma_kernel<BQ, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM);
        if (ce != cudaSuccess) return (int)ce;
        configured = true;
    }
    const int tiles = (max_rows + BQ - 1) / BQ;
    Params q = p;
    q.run_tiles = p.chunk / BQ > 0 && p.chunk / BQ < tiles ? p.chunk / BQ : 0;
    // (whole runs of tiles: those beyond the entry's last row have nothing to do)
    const int cols = q.run_tiles ? (tiles + q.run_tiles - 1) / q.run_tiles * q.run_tiles : tiles;
    const dim3 grid(cols, n_entries, C::ES * p.splits);
    cudaError_t le = p.splits == 1
        ? launch_kernel(attention_talk_mma_kernel<BQ, false>, grid, dim3(C::THREADS), C::SMEM, s, q)
        : launch_kernel(attention_talk_mma_kernel<BQ, true>, grid, dim3(C::THREADS), C::SMEM, s, q);
    if (le != cudaSuccess) return (int)le;
    if (p.splits > 1) {
        le = launch_kernel(attention_talk_merge_kernel, dim3((unsigned)((long long)p.n_rows * H)), dim3(128), 0, s,
                           (const float*)p.stats, (const float*)p.part, p.gate, p.gate_stride, p.out, p.out_stride, p.splits,
                           p.n_rows);
        if (le != cudaSuccess) return (int)le;
    }
    IB_LAUNCH_CHECK();
    return IB_OK;
}
}  // namespace

// What was compiled: sizes, then for eight queries a CTA (few = 0) or for few rows an entry (few = 1) the queries
// of a CTA, the keys of a tile, the blocks of the values, the bytes of shared memory, whether it can run.
IB_EXPORT int ib_attention_talk_mma_info(int what, int few) {
    using A = Cfg<8>;
    using B = Cfg<BQ_FEW>;
    const int v[] = {H, G, D, E, few ? BQ_FEW : 8, few ? B::BN : A::BN, few ? B::ES : A::ES, few ? B::SMEM : A::SMEM,
                     (few ? B::FITS : A::FITS) ? 1 : 0};
    return what >= 0 && what < 9 ? v[what] : -1;
}

IB_EXPORT long long ib_attention_talk_mma_scratch_bytes(int n_rows, int splits) {
    return (long long)splits * n_rows * H * (2 + E) * (long long)sizeof(float);
}

// q rows begin with H * D queries (row stride q_stride), out rows hold H * E (stride out_stride); talk float32 [H, H]
// whose values are exact in bf16, or null; gate bf16, one per (row, head), or null.
// max_rows: an upper bound on the rows of any entry (the grid's width); few: the variant for few rows an entry.
// splits > 1: the keys from the first that a CTA's first query sees, rounded down to the key tile, in slices of
// `slice_len` (a multiple of the key tile; together they must reach the last query) over that many CTAs, through
// `scratch`; n_rows: all rows.
IB_EXPORT int ib_attention_talk_mma(const void* q, int q_stride, const void* k_pool, const void* v_pool, void* out,
                                    int out_stride, const float* talk, const void* gate,
                                    int gate_stride, const int* cu_rows, const int* positions, const int* block_tables,
                                    int max_blocks, int n_entries, int max_rows, int page_size, int num_pages,
                                    int chunk, int window, unsigned* err, int n_rows, int few, int splits,
                                    int slice_len, void* scratch, long long scratch_bytes, void* stream) {
    if (n_entries <= 0 || max_rows <= 0 || n_rows <= 0) return IB_OK;
    if (!q || !k_pool || !v_pool || !out || !cu_rows || !positions || !block_tables || !err) return IB_ERR_BAD_ARG;
    if (page_size <= 0 || num_pages <= 0 || max_blocks <= 0 || chunk < 0 || window < 0 || splits < 1 ||
        q_stride < H * D || out_stride < H * E || (gate && gate_stride < H))
        return IB_ERR_BAD_ARG;
    if (q_stride % 8 || out_stride % 8 || (((uintptr_t)q | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)out) & 15))
        return IB_ERR_UNSUPPORTED;
    if (n_entries > 65535 || (long long)num_pages * G * page_size > 0x7fffffffLL) return IB_ERR_TOO_LARGE;
    if (splits > 1 && (!scratch || scratch_bytes < ib_attention_talk_mma_scratch_bytes(n_rows, splits))) return IB_ERR_BAD_ARG;
    Params p;
    p.q = (const bf16*)q;
    p.k_pool = (const bf16*)k_pool;
    p.v_pool = (const bf16*)v_pool;
    p.gate = (const bf16*)gate;
    p.out = (bf16*)out;
    p.talk = talk;
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
    p.run_tiles = 0;
    p.err = err;
    p.stats = (float*)scratch;
    p.part = scratch ? p.stats + (size_t)splits * n_rows * H * 2 : nullptr;
    return few ? launch_talk<BQ_FEW>(p, n_entries, max_rows, (cudaStream_t)stream)
               : launch_talk<8>(p, n_entries, max_rows, (cudaStream_t)stream);
}

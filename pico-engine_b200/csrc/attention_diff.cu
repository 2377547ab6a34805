// Differential attention over the paged bfloat16 cache: every head has two softmax maps, each with a query and a key of its own, over
// the same values; the head's output is the maps' difference a1 - lambda a2, divided by its root mean square.
//
//     a_m(i) = sum_j softmax_j(scale q_m(i) . k_m(j)) v(j),   o(i) = (a_1 - lambda a_2) / sqrt(mean((a_1 - lambda a_2)^2) + eps) * out_scale
//
// One block works on both maps of the same rows, so that a page's values are read once for both and the difference, its norm and the
// store need no second pass: warps 0-3 take the first map, warps 4-7 the second (mma.sync m16n8k16, float32 accumulators, S and P in
// registers, the C fragment of S reused as the A fragment of P V).  Key pages of both maps and the value page they share are copied
// to shared memory by cp.async, the next pages while one is multiplied.
//
//   prompt         a block = 64 consecutive tokens of one sequence (16 a warp) x one head; the second map's warps hand their normalised
//                  outputs to the first map's through shared memory, which finish the rows.
//   single tokens  a block = one token x one key/value head (the heads that share it, 16 a row tile) x a range of the token's pages; a warp
//                  takes 16 keys of every page.  The ranges of a (token, key/value head) are one thread-block cluster: each merges its warps'
//                  (max, sum, output), and the cluster's blocks finish a head each in turn from one another's results through distributed
//                  shared memory.  Pages that hold nothing new are asked for before the kernel waits for its predecessor, which can have
//                  written each token's own row only.
//
// Head sizes: D a multiple of 16 up to 256, Dv a multiple of 8 up to 256.  Queries lie key/value head by key/value head as
// [map 1 of its heads | map 2 of its heads]; the key pool has two heads (one a map) and the value pool one per key/value head.
#include "common.cuh"
#include <map>
#include <mutex>
#include <tuple>

#define DA_THREADS 256
#define DA_PAD 8
#define DA_ROWS 64                                // tokens of a prompt block
#define DA_MAX_SPLITS 16

struct DiffArgs {
    const bf16* q; int q_stride;
    const bf16* k_pool; const bf16* v_pool;
    const int* table; int table_stride;
    const int* tok_pos; const int* tok_row;
    const int* tiles;                             // prompt: runs of at most 64 tokens (row, first token, tokens, first position)
    int H, G, D, Dv, window; float scale, lambda, eps, out_scale;
    bf16* out; int out_ld, out_col;
    int splits;
};

__device__ __forceinline__ void da_ldsm_x4(uint32_t (&r)[4], const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void da_ldsm_x4_trans(uint32_t (&r)[4], uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void da_ldsm_x2_trans(uint32_t (&r)[2], const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a));
}
__device__ __forceinline__ void da_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void da_cp16(void* dst, const void* src, int bytes) {      // 16 bytes global -> shared; `bytes` 0 writes zeros
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" :: "r"(d), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void da_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void da_wait() { asm volatile("cp.async.wait_group %0;" :: "n"(N) : "memory"); }
__device__ __forceinline__ float da_exp2(float v) {                                    // 2^v; 2^-inf = 0
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
__device__ __forceinline__ uint32_t da_pack(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ void da_cluster_sync() {
    asm volatile("barrier.cluster.arrive.release;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire;" ::: "memory");
}
__device__ __forceinline__ unsigned da_cluster_rank() {
    unsigned r;
    asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}
__device__ __forceinline__ float da_ld_cluster(const float* local, unsigned rank) {    // the float at the same place of block `rank` of the cluster
    unsigned a = (unsigned)__cvta_generic_to_shared(local), r;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(a), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(r) : "memory");
    return v;
}

// DKM: most 16-wide steps of D; NVM: most 8-wide value tiles; NS: stages of pages in shared memory.
template <int DKM, int NVM, int NS, bool PROMPT>
__global__ void __launch_bounds__(DA_THREADS) attention_diff_kernel(DiffArgs a) {
    constexpr int NT = PROMPT ? 8 : 2;                                                 // tiles of 8 keys a warp takes of a page
    pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char da_smem[];
    __shared__ float red[33];
    const int D = a.D, Dv = a.Dv, G = a.G, per = a.H / G;
    const int kp = D + DA_PAD, vp = Dv + DA_PAD, dk = D >> 4, nv = Dv >> 3;
    const int stage_elems = PE_PAGE * (2 * kp + vp);                                   // K of map 1 [64][kp], K of map 2, V [64][vp]
    bf16* stages = reinterpret_cast<bf16*>(da_smem);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, map = warp >> 2, w4 = warp & 3;

    int seq, p_first, p_last, g, row0 = 0, n_rows;                                     // row0: first head of this block's row tile within the group
    int tok[2], head[2], qpos[2];
    bool live[2];
    if (PROMPT) {
        const int* r = a.tiles + 4 * blockIdx.y;
        const int h = blockIdx.x;
        g = h / per; seq = r[0]; n_rows = r[2]; p_first = r[3]; p_last = r[3] + r[2] - 1;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int i = w4 * 16 + (lane >> 2) + x * 8;
            live[x] = i < n_rows; tok[x] = r[1] + i; head[x] = h % per; qpos[x] = p_first + i;
        }
    } else {
        const int tiles_per = (per + 15) >> 4, t = blockIdx.z;
        g = blockIdx.y / tiles_per; row0 = (blockIdx.y % tiles_per) * 16; n_rows = min(16, per - row0);
        seq = a.tok_row[t]; p_first = p_last = a.tok_pos[t];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int i = (lane >> 2) + x * 8;
            live[x] = i < n_rows; tok[x] = t; head[x] = row0 + i; qpos[x] = p_first;
        }
    }
    const int page_lo = (a.window > 0 && p_first - a.window + 1 > 0) ? (p_first - a.window + 1) / PE_PAGE : 0;
    const int page_hi = p_last / PE_PAGE;
    int b_begin = page_lo, b_end = page_hi + 1;
    if (!PROMPT && a.splits > 1) {
        const int per_split = (page_hi - page_lo + a.splits) / a.splits;
        b_begin = page_lo + (int)blockIdx.x * per_split;
        b_end = min(page_hi + 1, b_begin + per_split);
    }
    const int k_end = p_last + 1;
    const int* table = a.table + (size_t)seq * a.table_stride;

    // copies of one page: a thread's 16-byte units are DA_THREADS apart, their (row, column) advance by fixed steps
    const int kper = D >> 3, vper = Dv >> 3;
    const int k_r0 = tid / kper, k_c0 = tid % kper, k_dr = DA_THREADS / kper, k_dc = DA_THREADS % kper;
    const int v_r0 = tid / vper, v_c0 = tid % vper, v_dr = DA_THREADS / vper, v_dc = DA_THREADS % vper;
    auto copy_page = [&](int blk, int stage) {
        const int page = table[blk];
        const int valid = page >= 0 ? min(PE_PAGE, k_end - blk * PE_PAGE) : 0;
        bf16* ks = stages + (size_t)stage * stage_elems;
        bf16* vs = ks + 2 * PE_PAGE * kp;
        // the key pages of a group's two maps are neighbours in the pool: 128 rows of D
        const bf16* ksrc = a.k_pool + ((size_t)max(page, 0) * 2 * G + 2 * g) * PE_PAGE * D;
        for (int r = k_r0, c = k_c0; r < 2 * PE_PAGE;) {
            da_cp16(ks + (size_t)r * kp + c * 8, ksrc + (size_t)r * D + c * 8, (r & (PE_PAGE - 1)) < valid ? 16 : 0);
            r += k_dr; c += k_dc;
            if (c >= kper) { c -= kper; ++r; }
        }
        const bf16* vsrc = a.v_pool + ((size_t)max(page, 0) * G + g) * PE_PAGE * Dv;
        for (int r = v_r0, c = v_c0; r < PE_PAGE;) {
            da_cp16(vs + (size_t)r * vp + c * 8, vsrc + (size_t)r * Dv + c * 8, r < valid ? 16 : 0);
            r += v_dr; c += v_dc;
            if (c >= vper) { c -= vper; ++r; }
        }
    };
    bool waited = PROMPT;
    if (PROMPT) pdl_wait();
#pragma unroll
    for (int s = 0; s < NS - 1; ++s) {
        const int blk = b_begin + s;
        if (blk < b_end) {
            if (!waited && blk == page_hi) { pdl_wait(); waited = true; }              // the page with the token's own row
            copy_page(blk, s);
        }
        da_commit();
    }
    if (!waited) pdl_wait();

    uint32_t qf[DKM][4];
#pragma unroll
    for (int kk = 0; kk < DKM; ++kk) {
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int rr = x & 1, col = kk * 16 + (lane & 3) * 2 + (x >> 1) * 8;
            qf[kk][x] = (kk < dk && live[rr]) ? *reinterpret_cast<const uint32_t*>(a.q + (size_t)tok[rr] * a.q_stride + ((size_t)(2 * g + map) * per + head[rr]) * D + col) : 0u;
        }
    }
    float o[NVM][4];
#pragma unroll
    for (int n = 0; n < NVM; ++n) { o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f; }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    const float sl2 = a.scale * 1.4426950408889634f;
    const int koff = PROMPT ? 0 : w4 * 16;
    const bool warp_live = !PROMPT || w4 * 16 < n_rows;
    const int q_first = PROMPT ? p_first + w4 * 16 : p_first, q_last = PROMPT ? min(p_last, q_first + 15) : p_first;

#pragma unroll 1
    for (int blk = b_begin; blk < b_end; ++blk) {
        const int i = blk - b_begin, stage = i % NS;
        if (blk + NS - 1 < b_end) copy_page(blk + NS - 1, (i + NS - 1) % NS);
        da_commit();
        da_wait<NS - 1>();
        __syncthreads();                                                               // this page's copies of all threads have landed
        const int kb = blk * PE_PAGE, valid = table[blk] >= 0 ? min(PE_PAGE, k_end - kb) : 0;
        // a warp whose rows see nothing of the page passes it by
        const bool any = warp_live && valid > 0 && kb + koff <= q_last && (a.window <= 0 || kb + koff + 8 * NT - 1 > q_first - a.window);
        if (any) {
            const bf16* k_s = stages + (size_t)stage * stage_elems + (size_t)map * PE_PAGE * kp;
            const bf16* v_s = stages + (size_t)stage * stage_elems + 2 * PE_PAGE * kp;
            const bf16* k_lane = k_s + (size_t)(koff + (lane & 7) + ((lane >> 4) << 3)) * kp + ((lane >> 3) & 1) * 8;
            const bf16* v_lane = v_s + (size_t)(koff + (lane & 15)) * vp + (lane >> 4) * 8;
            float s[NT][4];
#pragma unroll
            for (int n = 0; n < NT; ++n) { s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f; }
#pragma unroll
            for (int kk = 0; kk < DKM; ++kk) {
                if (kk < dk) {
#pragma unroll
                    for (int n = 0; n < NT; n += 2) {
                        uint32_t b[4];
                        da_ldsm_x4(b, k_lane + n * 8 * kp + kk * 16);
                        da_mma(s[n], qf[kk], b[0], b[1]);
                        da_mma(s[n + 1], qf[kk], b[2], b[3]);
                    }
                }
            }
            float mx[2] = {-INFINITY, -INFINITY};
            if (valid == PE_PAGE && kb + PE_PAGE - 1 <= q_first && (a.window <= 0 || kb > q_last - a.window)) {
#pragma unroll
                for (int n = 0; n < NT; ++n) {
#pragma unroll
                    for (int x = 0; x < 4; ++x) { s[n][x] *= sl2; mx[x >> 1] = fmaxf(mx[x >> 1], s[n][x]); }
                }
            } else {
#pragma unroll
                for (int n = 0; n < NT; ++n) {
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        const int rr = x >> 1, j = koff + n * 8 + (lane & 3) * 2 + (x & 1), key = kb + j;
                        const bool seen = j < valid && key <= qpos[rr] && (a.window <= 0 || qpos[rr] - key < a.window);
                        s[n][x] = seen ? s[n][x] * sl2 : -INFINITY;
                        mx[rr] = fmaxf(mx[rr], s[n][x]);
                    }
                }
            }
            float alpha[2];
#pragma unroll
            for (int rr = 0; rr < 2; ++rr) {
                mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 1));
                mx[rr] = fmaxf(mx[rr], __shfl_xor_sync(0xffffffffu, mx[rr], 2));
                const float m_new = fmaxf(m[rr], mx[rr]);
                alpha[rr] = m[rr] > -INFINITY ? da_exp2(m[rr] - m_new) : 1.f;
                m[rr] = m_new;
                l[rr] *= alpha[rr];
            }
            const float m0 = m[0] > -INFINITY ? m[0] : 0.f, m1 = m[1] > -INFINITY ? m[1] : 0.f;
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                s[n][0] = da_exp2(s[n][0] - m0); s[n][1] = da_exp2(s[n][1] - m0);
                s[n][2] = da_exp2(s[n][2] - m1); s[n][3] = da_exp2(s[n][3] - m1);
                l[0] += s[n][0] + s[n][1];
                l[1] += s[n][2] + s[n][3];
            }
            if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
                for (int n = 0; n < NVM; ++n) { o[n][0] *= alpha[0]; o[n][1] *= alpha[0]; o[n][2] *= alpha[1]; o[n][3] *= alpha[1]; }
            }
#pragma unroll
            for (int ks = 0; ks < NT / 2; ++ks) {
                uint32_t pf[4] = {da_pack(s[2 * ks][0], s[2 * ks][1]), da_pack(s[2 * ks][2], s[2 * ks][3]),
                                  da_pack(s[2 * ks + 1][0], s[2 * ks + 1][1]), da_pack(s[2 * ks + 1][2], s[2 * ks + 1][3])};
                const uint32_t v_at = (uint32_t)__cvta_generic_to_shared(v_lane + (size_t)ks * 16 * vp);
#pragma unroll
                for (int n = 0; n < NVM; n += 2) {
                    if (n + 1 < nv) {                                                  // two tiles of 8 value columns at once
                        uint32_t b[4];
                        da_ldsm_x4_trans(b, v_at + n * 16);
                        da_mma(o[n], pf, b[0], b[1]);
                        da_mma(o[n + 1], pf, b[2], b[3]);
                    } else if (n < nv) {
                        uint32_t b[2];
                        da_ldsm_x2_trans(b, v_s + (size_t)(koff + ks * 16 + (lane & 15)) * vp + n * 8);
                        da_mma(o[n], pf, b[0], b[1]);
                    }
                }
            }
        }
        __syncthreads();                                                               // the stage is free for another page
    }
#pragma unroll
    for (int rr = 0; rr < 2; ++rr) {
        l[rr] += __shfl_xor_sync(0xffffffffu, l[rr], 1);
        l[rr] += __shfl_xor_sync(0xffffffffu, l[rr], 2);
    }
    da_wait<0>();
    __syncthreads();                                                                   // from here on the stages' memory holds results
    float* res = reinterpret_cast<float*>(da_smem);
    const int c0 = (lane & 3) * 2, r0 = lane >> 2;

    if constexpr (PROMPT) {
        const int op = Dv + 4;                                                         // floats between rows (skews the banks)
        const float inv[2] = {l[0] > 0.f ? 1.0f / l[0] : 0.f, l[1] > 0.f ? 1.0f / l[1] : 0.f};
        if (map == 1) {
#pragma unroll
            for (int n = 0; n < NVM; ++n)
                if (n < nv) {
#pragma unroll
                    for (int rr = 0; rr < 2; ++rr)
                        *reinterpret_cast<float2*>(res + (size_t)(w4 * 16 + r0 + rr * 8) * op + n * 8 + c0) =
                            make_float2(o[n][2 * rr] * inv[rr] * a.lambda, o[n][2 * rr + 1] * inv[rr] * a.lambda);
                }
        }
        __syncthreads();
        if (map == 1) return;
        float ss[2] = {0.f, 0.f};
#pragma unroll
        for (int n = 0; n < NVM; ++n)
            if (n < nv) {
#pragma unroll
                for (int rr = 0; rr < 2; ++rr) {
                    const float2 b = *reinterpret_cast<const float2*>(res + (size_t)(w4 * 16 + r0 + rr * 8) * op + n * 8 + c0);
                    o[n][2 * rr] = o[n][2 * rr] * inv[rr] - b.x;
                    o[n][2 * rr + 1] = o[n][2 * rr + 1] * inv[rr] - b.y;
                    ss[rr] = fmaf(o[n][2 * rr], o[n][2 * rr], ss[rr]);
                    ss[rr] = fmaf(o[n][2 * rr + 1], o[n][2 * rr + 1], ss[rr]);
                }
            }
#pragma unroll
        for (int rr = 0; rr < 2; ++rr) {
            ss[rr] += __shfl_xor_sync(0xffffffffu, ss[rr], 1);
            ss[rr] += __shfl_xor_sync(0xffffffffu, ss[rr], 2);
            const float f = 1.0f / sqrtf(ss[rr] / (float)Dv + a.eps) * a.out_scale;
            if (!live[rr]) continue;
            bf16* dst = a.out + (size_t)tok[rr] * a.out_ld + a.out_col + (size_t)blockIdx.x * Dv + c0;
#pragma unroll
            for (int n = 0; n < NVM; ++n)
                if (n < nv) *reinterpret_cast<__nv_bfloat162*>(dst + n * 8) = __floats2bfloat162_rn(o[n][2 * rr] * f, o[n][2 * rr + 1] * f);
        }
        return;
    } else {
        // the warps' results: [8][n_rows][Dv] outputs, [8][16] maxima and sums; then the block's: [2][n_rows][Dv], [2][16], [2][16]
        float* wm = res;
        float* wl = wm + 8 * 16;
        float* bm = wl + 8 * 16;                                                       // the block's maxima, sums and outputs, which the cluster reads
        float* bl = bm + 2 * 16;
        float* bo = bl + 2 * 16;
        float* wo = bo + (size_t)2 * n_rows * Dv;
#pragma unroll
        for (int rr = 0; rr < 2; ++rr) {
            if (!live[rr]) continue;
            const int row = r0 + rr * 8;
            if ((lane & 3) == 0) { wm[warp * 16 + row] = m[rr]; wl[warp * 16 + row] = l[rr]; }
            float* dst = wo + ((size_t)warp * n_rows + row) * Dv + c0;
#pragma unroll
            for (int n = 0; n < NVM; ++n)
                if (n < nv) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[n][2 * rr], o[n][2 * rr + 1]);
        }
        __syncthreads();
        for (int e = tid; e < 2 * n_rows * Dv; e += DA_THREADS) {
            const int mp = e / (n_rows * Dv), row = (e / Dv) % n_rows, d = e % Dv;
            float M = -INFINITY;
#pragma unroll
            for (int w = 0; w < 4; ++w) M = fmaxf(M, wm[(mp * 4 + w) * 16 + row]);
            float acc = 0.f, den = 0.f;
            if (M > -INFINITY) {
#pragma unroll
                for (int w = 0; w < 4; ++w) {
                    const float f = da_exp2(wm[(mp * 4 + w) * 16 + row] - M);
                    acc = fmaf(f, wo[((size_t)(mp * 4 + w) * n_rows + row) * Dv + d], acc);
                    den = fmaf(f, wl[(mp * 4 + w) * 16 + row], den);
                }
            }
            bo[e] = acc;
            if (d == 0) { bm[mp * 16 + row] = M; bl[mp * 16 + row] = den; }
        }
        const int S = a.splits;
        const unsigned rank = S > 1 ? da_cluster_rank() : 0u;
        if (S > 1) da_cluster_sync(); else __syncthreads();
        float* fin = wo;                                                               // [2][Dv]: the finished maps of one head (the warps' outputs are done with)
        for (int row = rank; row < n_rows; row += S) {
            for (int e = tid; e < 2 * Dv; e += DA_THREADS) {
                const int mp = e / Dv, d = e % Dv;
                float acc = 0.f, den = 0.f;
                if (S > 1) {
                    float ms[DA_MAX_SPLITS], M = -INFINITY;
#pragma unroll
                    for (int c = 0; c < DA_MAX_SPLITS; ++c) { ms[c] = c < S ? da_ld_cluster(bm + mp * 16 + row, c) : -INFINITY; M = fmaxf(M, ms[c]); }
#pragma unroll
                    for (int c = 0; c < DA_MAX_SPLITS; ++c)
                        if (c < S && ms[c] > -INFINITY) {
                            const float f = da_exp2(ms[c] - M);
                            acc = fmaf(f, da_ld_cluster(bo + ((size_t)mp * n_rows + row) * Dv + d, c), acc);
                            den = fmaf(f, da_ld_cluster(bl + mp * 16 + row, c), den);
                        }
                } else { acc = bo[((size_t)mp * n_rows + row) * Dv + d]; den = bl[mp * 16 + row]; }
                fin[e] = den > 0.f ? acc / den : 0.f;
            }
            __syncthreads();
            float v = 0.f;
            if (tid < Dv) v = fin[tid] - a.lambda * fin[Dv + tid];                     // (Dv is at most the number of threads)
            const float f = 1.0f / sqrtf(block_sum(v * v, red) / (float)Dv + a.eps) * a.out_scale;
            if (tid < Dv) a.out[(size_t)blockIdx.z * a.out_ld + a.out_col + (size_t)(g * per + row0 + row) * Dv + tid] = __float2bfloat16_rn(v * f);
            __syncthreads();
        }
        if (S > 1) da_cluster_sync();                                                  // nobody leaves while its results are still being read
    }
}

namespace {

size_t da_stage_bytes(int D, int Dv) { return 2 * (size_t)PE_PAGE * (2 * (D + DA_PAD) + Dv + DA_PAD); }
size_t da_result_bytes(int rows, int Dv, bool prompt) {
    return 4 * (prompt ? (size_t)DA_ROWS * (Dv + 4) : 2 * 8 * 16 + 2 * 2 * 16 + (size_t)10 * rows * Dv);
}
size_t da_smem_bytes(int D, int Dv, int rows, int NS, bool prompt) {
    const size_t a = NS * da_stage_bytes(D, Dv), b = da_result_bytes(rows, Dv, prompt);
    return a > b ? a : b;
}

std::mutex da_mu;
std::map<std::tuple<const void*, size_t, int>, int> da_clusters;

// how many clusters of `splits` blocks of this kernel can be resident at once
int da_max_clusters(const void* fn, size_t smem, int splits) {
    std::lock_guard<std::mutex> lock(da_mu);
    const auto key = std::make_tuple(fn, smem, splits);
    const auto it = da_clusters.find(key);
    if (it != da_clusters.end()) return it->second;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(splits); cfg.blockDim = dim3(DA_THREADS); cfg.dynamicSmemBytes = smem;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = splits; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr; cfg.numAttrs = 1;
    int n = 0;
    if (cudaOccupancyMaxActiveClusters(&n, fn, &cfg) != cudaSuccess) { cudaGetLastError(); n = 0; }
    da_clusters[key] = n;
    return n;
}

template <int DKM, int NVM, int NS>
int da_prompt(const DiffArgs& a, int n_runs, size_t smem, cudaStream_t s) {
    PE_TRY(cudaFuncSetAttribute(attention_diff_kernel<DKM, NVM, NS, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    PE_TRY(pe_launch(attention_diff_kernel<DKM, NVM, NS, true>, dim3(a.H, n_runs), DA_THREADS, smem, s, a));
    return 0;
}

template <int DKM, int NVM, int NS>
int da_single(DiffArgs a, int T, int pages, size_t smem, cudaStream_t s) {
    const auto kernel = attention_diff_kernel<DKM, NVM, NS, false>;
    PE_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    PE_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
    const int groups = a.G * ((a.H / a.G + 15) / 16);
    int splits = 1;
    // more ranges while they leave a block at least one page and all clusters can run at once
    while (splits < DA_MAX_SPLITS && 2 * splits <= pages && da_max_clusters((const void*)kernel, smem, 2 * splits) >= T * groups) splits *= 2;
    a.splits = splits;
    PE_TRY(pe_launch_cluster(kernel, dim3(splits, groups, T), DA_THREADS, smem, s, splits, a));
    return 0;
}

}  // namespace

extern "C" int pe_attention_diff_takes(int H, int G, int D, int Dv) {
    return H > 0 && G > 0 && H % G == 0 && D % 16 == 0 && D >= 16 && D <= 256 && Dv % 8 == 0 && Dv >= 8 && Dv <= 256;
}

// tiles null: single tokens (max_context bounds every token's position + 1 and fixes the launch shape); else prompt runs.
extern "C" int pe_attention_diff(const void* q, int q_stride, void* out, int out_ld, int out_col, const void* k_pool, const void* v_pool,
                                 const int* table, int table_stride, const int* tok_pos, const int* tok_row, const int* tiles, int n_runs,
                                 int T, int H, int G, int D, int Dv, int window, float scale, float lambda, float eps, float out_scale,
                                 int max_context, void* stream) {
    if (T <= 0) return 0;
    if (!pe_attention_diff_takes(H, G, D, Dv) || (tiles && (n_runs <= 0 || n_runs > 65535)) || T > 65535 || G * ((H / G + 15) / 16) > 65535) return PE_ERR_UNSUPPORTED;
    if (((uintptr_t)k_pool | (uintptr_t)v_pool) & 15 || ((uintptr_t)q | (uintptr_t)out) & 3 || (q_stride & 1) || (out_ld & 1) || (out_col & 1)) return PE_ERR_UNSUPPORTED;
    DiffArgs a = {(const bf16*)q, q_stride, (const bf16*)k_pool, (const bf16*)v_pool, table, table_stride, tok_pos, tok_row, tiles,
                  H, G, D, Dv, window, scale, lambda, eps, out_scale, (bf16*)out, out_ld, out_col, 1};
    cudaStream_t s = (cudaStream_t)stream;
    const bool prompt = tiles != nullptr;
    const int rows = H / G < 16 ? H / G : 16;
    const size_t limit = 220 * 1024;
    const bool three = !prompt && da_smem_bytes(D, Dv, rows, 3, prompt) <= limit;
    const size_t smem = da_smem_bytes(D, Dv, rows, three ? 3 : 2, prompt);
    if (smem > limit) return PE_ERR_UNSUPPORTED;
    int span = max_context > 0 ? max_context : 1;
    if (window > 0 && window + PE_PAGE - 1 < span) span = window + PE_PAGE - 1;
    const int pages = (span + PE_PAGE - 1) / PE_PAGE;
    int rc;
#define DA_RUN(DKM, NVM) (prompt ? da_prompt<DKM, NVM, 2>(a, n_runs, smem, s) : three ? da_single<DKM, NVM, 3>(a, T, pages, smem, s) : da_single<DKM, NVM, 2>(a, T, pages, smem, s))
    if (D <= 64) rc = Dv <= 128 ? DA_RUN(4, 16) : DA_RUN(4, 32);
    else if (D <= 128) rc = Dv <= 128 ? DA_RUN(8, 16) : DA_RUN(8, 32);
    else rc = Dv <= 128 ? DA_RUN(16, 16) : DA_RUN(16, 32);
#undef DA_RUN
    if (rc) return rc;
    PE_LAUNCH_CHECK();
    return 0;
}

// Differential attention of prompts on the 5th-generation tensor cores: heads of two softmax maps over the same values, whose output is
// the maps' difference divided by its root mean square (the equations stand in attention_diff.cu).  Both products of flash attention
// run as tcgen05.mma with their accumulators in tensor memory.
//
//   one CTA   = a run of up to 128 consecutive tokens of one sequence x one head, both maps
//   a step    = two pages of the cache (128 keys) for one map; the maps take turns, so that the tensor core works on one map's
//               products while the softmax warps work on the other's scores
//   warp 0      loader: TMA tiled loads (128-byte swizzle) of both maps' queries and, every second step, of two pages' keys of both
//               maps and of the values they share into a ring of two stages; it alone reads the page table
//   warp 1      allocates tensor memory (two S buffers and two accumulators of up to 128 columns: one of each a map); one lane
//               issues S = Q_m K_m^T and O_m += P V, S of the next step before P V of this one
//   warps 2-9   softmax, two threads a query row, one for each page of the step, with a running maximum and sum a map; at the end
//               each thread has half of both maps' rows in registers, forms the difference, meets its partner for the sum of
//               squares and stores its half
//
// Head sizes that are multiples of 8: D up to 64 (a key row's 64-column box is filled with zeros beyond D, so what the query box holds
// there does not count), Dv up to 128.  Every mbarrier wait is bounded (*status 5), as in attention_prefill_tcgen05.cu.
#include "tcgen05_attention.cuh"

#define DT_QTILE 128
#define DT_KTILE PE_PAGE
#define DT_STAGES 2                                // steps' keys and values in flight or in use
#define DT_THREADS 320                             // loader, MMA issuer, and two softmax warps for each 32 rows
#define DT_PANEL (2 * DT_KTILE * 128)              // 128 rows of 64 columns: one swizzled panel
#define DT_BAR_WORDS (13 + 2 * DT_STAGES)
#define DT_TMEM_COLS 512                           // S buffers at columns 0 and 128, O of the maps from columns 256 and 384
#define DT_O_COL 256
#define DT_LAZY 8.0f
#define DT_STAGE_BYTES(VP) ((2 + (VP)) * DT_PANEL) // keys of map 1, keys of map 2, values (VP panels)
#define DT_TILE_BYTES(VP) (2 * DT_PANEL + DT_STAGES * DT_STAGE_BYTES(VP) + 2 * 2 * DT_PANEL)      // queries of both maps, stages, two P tiles
#define DT_SMEM_BYTES(VP) (DT_TILE_BYTES(VP) + 8 * DT_BAR_WORDS + 8 * DT_STAGES + 2 * 2 * DT_QTILE * 4)

struct DtArgs {
    bf16* out; int out_ld, out_col;
    const int* block_table; int table_stride; const int4* tiles;
    int H, G, D, Dv, window; float scale_log2e, lambda, eps, out_scale;
    int k_rows, v_rows;                            // rows of the key and value pools seen as matrices [rows][head size]
};

// VP: 64-column panels of a value row.
template <int VP>
__global__ void __launch_bounds__(DT_THREADS, 1) attention_diff_tcgen05_kernel(const __grid_constant__ CUtensorMap map_q,
                                                                               const __grid_constant__ CUtensorMap map_k,
                                                                               const __grid_constant__ CUtensorMap map_v,
                                                                               const DtArgs p, int* status) {
    extern __shared__ __align__(1024) unsigned char dt_mem[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const unsigned q_s = at_smem(dt_mem), kv_s = q_s + 2 * DT_PANEL, p_s = kv_s + DT_STAGES * DT_STAGE_BYTES(VP);
    unsigned long long* bars = reinterpret_cast<unsigned long long*>(dt_mem + DT_TILE_BYTES(VP));
    unsigned long long &q_full = bars[0], &p_full = bars[1];
    unsigned long long *pv_done = bars + 2, *s_full = bars + 4, *s_free = bars + 6, *kv_full = bars + 8, *kv_empty = bars + 8 + DT_STAGES;
    unsigned long long* pair_bar = bars + 8 + 2 * DT_STAGES;       // one for the two softmax warps of each 32 rows
    unsigned& tmem_base_s = *reinterpret_cast<unsigned*>(bars + 12 + 2 * DT_STAGES);
    volatile unsigned* stage_flags = reinterpret_cast<volatile unsigned*>(bars + DT_BAR_WORDS);   // bit g: page g of the stage exists
    float* exchange = reinterpret_cast<float*>(bars + DT_BAR_WORDS + DT_STAGES);    // [meeting parity][half][row]: what the halves of a row tell each other
    if (q_s & 1023u) {                                              // every thread alike: nothing is allocated yet
        if (threadIdx.x == 0) atomicExch(status, 6);
        return;
    }
    if (threadIdx.x == 0) {
        asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(at_smem(&q_full)) : "memory");
        asm volatile("mbarrier.init.shared::cta.b64 [%0], 8;" ::"r"(at_smem(&p_full)) : "memory");          // the eight softmax warps
        for (int q = 0; q < 4; ++q) asm volatile("mbarrier.init.shared::cta.b64 [%0], 2;" ::"r"(at_smem(&pair_bar[q])) : "memory");
        for (int s = 0; s < DT_STAGES; ++s) {
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(at_smem(&kv_full[s])) : "memory");
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(at_smem(&kv_empty[s])) : "memory");
        }
        for (int b = 0; b < 2; ++b) {
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(at_smem(&s_full[b])) : "memory");
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 8;" ::"r"(at_smem(&s_free[b])) : "memory");
            asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(at_smem(&pv_done[b])) : "memory");
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(at_smem(&tmem_base_s)), "r"((unsigned)DT_TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const unsigned tmem = tmem_base_s;
    // only now may the next kernel of the stream be scheduled: it could take tensor memory that a CTA of this grid still waits for
    pdl_launch_dependents();
    pdl_wait();

    const int4 info = p.tiles[blockIdx.y];                          // heads vary fastest: the runs that see the most keys start first
    const int brow = info.x, tok0 = info.y, n = info.z, pos0 = info.w;
    const int per = p.H / p.G, h = blockIdx.x, g_kv = h / per;
    const int first_key = (p.window > 0 && pos0 - p.window + 1 > 0) ? pos0 - p.window + 1 : 0;
    const int page_lo = first_key / DT_KTILE, page_hi = (pos0 + n - 1) / DT_KTILE;
    const int n_pages = page_hi - page_lo + 1, n_steps = (n_pages + 1) / 2, n_its = 2 * n_steps;      // an iteration: one step of one map

    if (warp == 0) {
        if (lane == 0) {                                            // ---------------- loader
            const int* table = p.block_table + (size_t)brow * p.table_stride;
            asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(at_smem(&q_full)), "r"((unsigned)(2 * DT_PANEL)) : "memory");
#pragma unroll
            for (int m = 0; m < 2; ++m) at_tma_2d(q_s + m * DT_PANEL, &map_q, ((2 * g_kv + m) * per + h % per) * p.D, tok0, at_smem(&q_full));
            int page[2] = {table[page_lo], 1 < n_pages ? table[page_lo + 1] : -1};
            for (int st = 0; st < n_steps; ++st) {
                const int s = st % DT_STAGES;
                int next[2] = {-1, -1};                             // the step after this one: its entries travel during the wait
                if (2 * st + 2 < n_pages) next[0] = table[page_lo + 2 * st + 2];
                if (2 * st + 3 < n_pages) next[1] = table[page_lo + 2 * st + 3];
                if (st >= DT_STAGES && !at_wait(at_smem(&kv_empty[s]), (unsigned)((st / DT_STAGES) - 1) & 1u)) { atomicExch(status, 5); break; }
                const unsigned bar = at_smem(&kv_full[s]), k_dst = kv_s + s * DT_STAGE_BYTES(VP), v_dst = k_dst + 2 * DT_PANEL;
                stage_flags[s] = (page[0] >= 0 ? 1u : 0u) | (page[1] >= 0 ? 2u : 0u);
                asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"((unsigned)DT_STAGE_BYTES(VP)) : "memory");
#pragma unroll
                for (int g = 0; g < 2; ++g) {
                    // a page that is not there is read from beyond the pool's end, which gives zeros: its scores are masked and its
                    // values add nothing
#pragma unroll
                    for (int m = 0; m < 2; ++m)
                        at_tma_2d(k_dst + m * DT_PANEL + g * (DT_KTILE * 128), &map_k, 0,
                                  page[g] >= 0 ? ((page[g] * p.G + g_kv) * 2 + m) * DT_KTILE : p.k_rows, bar);
#pragma unroll
                    for (int c = 0; c < VP; ++c)
                        at_tma_2d(v_dst + c * DT_PANEL + g * (DT_KTILE * 128), &map_v, 64 * c, page[g] >= 0 ? (page[g] * p.G + g_kv) * DT_KTILE : p.v_rows, bar);
                }
                page[0] = next[0]; page[1] = next[1];
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {                                            // ---------------- MMA issuer
            // instruction descriptors: float32 accumulator, bfloat16 operands, M = 128; S: A and B K-major, N = 128 keys;
            // O: B MN-major (bit 16), N = Dv rounded up to 16
            const unsigned idesc_s = (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned)((2 * DT_KTILE) >> 3) << 17) | ((unsigned)(DT_QTILE >> 4) << 24);
            const unsigned idesc_o = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((unsigned)(((p.Dv + 15) & ~15) >> 3) << 17) | ((unsigned)(DT_QTILE >> 4) << 24);
            const unsigned long long dq = at_desc(q_s, 0, 1024), dk = at_desc(kv_s, 0, 1024), dp = at_desc(p_s, 0, 1024);
            const unsigned long long dv = at_desc(kv_s + 2 * DT_PANEL, DT_PANEL, 1024);
            const int k_steps = (p.D + 15) >> 4;
            bool ok = at_wait(at_smem(&q_full), 0u);
            auto issue_s = [&](int it) -> bool {                    // S of iteration `it` (map it & 1) into S buffer it & 1
                const int st = it >> 1, s = st % DT_STAGES, b = it & 1;
                if (!at_wait(at_smem(&kv_full[s]), (unsigned)(st / DT_STAGES) & 1u)) return false;
                if (it >= 2 && !at_wait(at_smem(&s_free[b]), (unsigned)((it >> 1) - 1) & 1u)) return false;
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const unsigned long long dqs = dq + (unsigned long long)(b * (DT_PANEL >> 4));
                const unsigned long long dks = dk + (unsigned long long)(s * (DT_STAGE_BYTES(VP) >> 4) + b * (DT_PANEL >> 4));
                for (int kk = 0; kk < k_steps; ++kk)                // 16 columns = 32 bytes inside the swizzle atom
                    at_mma(tmem + b * (2 * DT_KTILE), dqs + kk * 2, dks + kk * 2, idesc_s, kk > 0 ? 1u : 0u);
                at_commit(at_smem(&s_full[b]));
                return true;
            };
            if (ok) ok = issue_s(0);
            for (int it = 0; it < n_its && ok; ++it) {
                if (it + 1 < n_its && !issue_s(it + 1)) { ok = false; break; }
                const int s = (it >> 1) % DT_STAGES, b = it & 1;
                if (!at_wait(at_smem(&p_full), (unsigned)it & 1u)) { ok = false; break; }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const unsigned long long dps = dp + (unsigned long long)(b * (2 * DT_PANEL >> 4)), dvs = dv + (unsigned long long)(s * (DT_STAGE_BYTES(VP) >> 4));
#pragma unroll
                for (int kk = 0; kk < 2 * DT_KTILE / 16; ++kk) {    // 16 keys: 32 bytes further in P's rows (64 keys a panel), 16 rows further in V
                    const unsigned off_p = ((kk / 4) * DT_PANEL + (kk % 4) * 32) >> 4, off_v = (kk * 16 * 128) >> 4;
                    at_mma(tmem + DT_O_COL + b * 128, dps + off_p, dvs + off_v, idesc_o, (it > 1 || kk > 0) ? 1u : 0u);
                }
                if (it & 1) at_commit(at_smem(&kv_empty[s]));       // both maps have read the stage
                at_commit(at_smem(&pv_done[b]));                    // and O of this map holds this step's share
            }
            if (!ok) atomicExch(status, 5);
        }
    } else {                                                        // ---------------- softmax, warps 2..9
        const int quarter = warp & 3;                               // the 32 lanes of tensor memory this warp may touch
        const int g = (warp - 2) >> 2;
        const int r = quarter * 32 + lane;                          // this thread's query row
        const int p_r = pos0 + r;
        const unsigned lane_addr = tmem + ((unsigned)(quarter * 32) << 16);
        const unsigned o_addr = lane_addr + DT_O_COL + g * (VP * 32);
        const unsigned pair = at_smem(&pair_bar[quarter]);
        float m_run = -INFINITY, l_run = 0.f, m_alt = -INFINITY, l_alt = 0.f;      // of this iteration's map and of the other
        bool ok = true;
        int it = 0, met = 0;                                        // met: how often the row's two threads have met
        auto swap = [&](float mine, float& theirs) -> bool {        // tell the other half `mine`, learn what it tells
            float* slot = exchange + (met & 1) * (2 * DT_QTILE);
            slot[g * DT_QTILE + r] = mine;
            __syncwarp();
            if (lane == 0) at_arrive(pair);
            if (!at_wait_warp(pair, (unsigned)met & 1u)) return false;
            theirs = slot[(g ^ 1) * DT_QTILE + r];
            ++met;
            return true;
        };
#pragma unroll 1
        for (; it < n_its; ++it) {
            const int b = it & 1, st = it >> 1, s_at = st % DT_STAGES;
            if (!at_wait_warp(at_smem(&kv_full[s_at]), (unsigned)(st / DT_STAGES) & 1u)) { ok = false; break; }   // the loader's flags
            const bool there = (stage_flags[s_at] >> g) & 1u;
            if (!at_wait_warp(at_smem(&s_full[b]), (unsigned)(it >> 1) & 1u)) { ok = false; break; }
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            const int key0 = (page_lo + 2 * st + g) * DT_KTILE;
            unsigned raw[DT_KTILE];
            at_ld32_start(lane_addr + b * (2 * DT_KTILE) + g * DT_KTILE, raw);
            at_ld32_start(lane_addr + b * (2 * DT_KTILE) + g * DT_KTILE + 32, raw + 32);
            at_ld_wait();
            at_pin32(raw); at_pin32(raw + 32);
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) at_arrive(at_smem(&s_free[b]));          // the buffer may take the map's next S
            float s[DT_KTILE];
#pragma unroll
            for (int c = 0; c < DT_KTILE; ++c) s[c] = __uint_as_float(raw[c]);
            const bool whole = there && key0 + DT_KTILE - 1 <= p_r && (p.window <= 0 || key0 > p_r - p.window);
            if (!whole) {
#pragma unroll
                for (int c = 0; c < DT_KTILE; ++c) {
                    const int key = key0 + c;
                    if (!there || key > p_r || (p.window > 0 && key <= p_r - p.window)) s[c] = -INFINITY;
                }
            }
            float mx[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
            for (int c = 4; c < DT_KTILE; ++c) mx[c & 3] = fmaxf(mx[c & 3], s[c]);
            const float m_mine = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
            float m_theirs;
            if (!swap(m_mine, m_theirs)) { ok = false; break; }
            // the reference point follows the row's maximum only when that has grown by more than DT_LAZY powers of two
            const float m_tile = fmaxf(m_mine, m_theirs) * p.scale_log2e;
            const float m_new = (m_run != -INFINITY && m_tile <= m_run + DT_LAZY) ? m_run : fmaxf(m_run, m_tile);
            const float m_use = m_new == -INFINITY ? 0.f : m_new;
            const float alpha = m_run == -INFINITY ? 1.0f : at_exp2(m_run - m_use);
            m_run = m_new;
            float sum[4] = {0.f, 0.f, 0.f, 0.f};
            unsigned packed[DT_KTILE / 2];
#pragma unroll
            for (int c = 0; c < DT_KTILE; c += 2) {
                const float e0 = at_exp2(fmaf(s[c], p.scale_log2e, -m_use)), e1 = at_exp2(fmaf(s[c + 1], p.scale_log2e, -m_use));
                sum[c & 3] += e0; sum[(c + 1) & 3] += e1;
                packed[c >> 1] = at_pack(e0, e1);
            }
            l_run = l_run * alpha + ((sum[0] + sum[1]) + (sum[2] + sum[3]));
            // the map's P tile is free, and its O holds every earlier step, once P.V of the iteration before last is done
            if (it >= 2) {
                if (!at_wait_warp(at_smem(&pv_done[b]), (unsigned)((it >> 1) - 1) & 1u)) { ok = false; break; }
                if (__any_sync(0xffffffffu, alpha != 1.0f)) {       // a row's reference point moved: rescale this half of the warp's rows of O
                    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll 1
                    for (int c = 0; c < VP * 32; c += 32) {
                        float o[32];
                        at_ld32(o_addr + b * 128 + c, o);
#pragma unroll
                        for (int i = 0; i < 32; ++i) o[i] *= alpha;
                        at_st32(o_addr + b * 128 + c, o);
                    }
                    asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
                }
            }
            unsigned char* p_row = dt_mem + (p_s - q_s) + b * (2 * DT_PANEL) + g * DT_PANEL + r * 128;
#pragma unroll
            for (int c = 0; c < DT_KTILE / 8; ++c)
                *reinterpret_cast<uint4*>(p_row + ((c ^ (r & 7)) << 4)) = make_uint4(packed[4 * c], packed[4 * c + 1], packed[4 * c + 2], packed[4 * c + 3]);
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // P is read by the tensor core's proxy
            asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
            __syncwarp();
            if (lane == 0) at_arrive(at_smem(&p_full));
            const float tm = m_run, tl = l_run;
            m_run = m_alt; l_run = l_alt; m_alt = tm; l_alt = tl;
        }
        // an even number of iterations: m_run, l_run are the first map's again.  The rows' sums, then the last P.V (products complete in
        // the order they were issued).
        float l1 = 0.f, l2 = 0.f;
        if (ok && !swap(l_run, l1)) ok = false;
        if (ok && !swap(l_alt, l2)) ok = false;
        if (ok && !at_wait_warp(at_smem(&pv_done[1]), (unsigned)(n_steps - 1) & 1u)) ok = false;
        if (ok) {
            asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
            l1 = g == 0 ? l_run + l1 : l1 + l_run;                  // the same sums in both threads
            l2 = g == 0 ? l_alt + l2 : l2 + l_alt;
            const float f1 = l1 > 0.f ? 1.0f / l1 : 0.f, f2 = l2 > 0.f ? p.lambda / l2 : 0.f;
            const int col0 = g * (VP * 32);
            float d[VP * 32], ss = 0.f;
#pragma unroll
            for (int c = 0; c < VP * 32; c += 32) {
                float o[32];
                at_ld32(o_addr + c, o);
#pragma unroll
                for (int i = 0; i < 32; ++i) d[c + i] = o[i] * f1;
                at_ld32(o_addr + 128 + c, o);
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    d[c + i] = col0 + c + i < p.Dv ? fmaf(-f2, o[i], d[c + i]) : 0.f;      // (columns beyond Dv hold nothing)
                    ss = fmaf(d[c + i], d[c + i], ss);
                }
            }
            float ss_theirs;
            if (!swap(ss, ss_theirs)) ok = false;
            else if (r < n) {
                const float f = 1.0f / sqrtf((g == 0 ? ss + ss_theirs : ss_theirs + ss) / (float)p.Dv + p.eps) * p.out_scale;
                bf16* o_row = p.out + (size_t)(tok0 + r) * p.out_ld + p.out_col + (size_t)h * p.Dv + col0;
#pragma unroll
                for (int i = 0; i < VP * 32; i += 8)
                    if (col0 + i < p.Dv)
                        *reinterpret_cast<uint4*>(o_row + i) = make_uint4(at_pack(d[i] * f, d[i + 1] * f), at_pack(d[i + 2] * f, d[i + 3] * f),
                                                                          at_pack(d[i + 4] * f, d[i + 5] * f), at_pack(d[i + 6] * f, d[i + 7] * f));
            }
        }
        if (!ok) atomicExch(status, 5);
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((unsigned)DT_TMEM_COLS) : "memory");
    }
}

extern "C" int pe_attention_diff_tcgen05_takes(int H, int G, int D, int Dv) {
    return H > 0 && G > 0 && H % G == 0 && D % 8 == 0 && D >= 8 && D <= 64 && Dv % 8 == 0 && Dv >= 8 && Dv <= 128;
}

// q: [n_tokens][q_stride], queries key/value head by key/value head as [map 1 of its heads | map 2]; k_pool [pages][2 G][64][D], v_pool
// [pages][G][64][Dv]; runs `tiles` of at most 128 tokens; out [n_tokens][out_ld], head h at column out_col + h * Dv.
extern "C" int pe_attention_diff_tcgen05(const void* q, int q_stride, void* out, int out_ld, int out_col, const void* k_pool, const void* v_pool,
                                         long long pool_pages, const int* table, int table_stride, const void* tiles, int n_tiles, int n_tokens,
                                         int H, int G, int D, int Dv, int window, float scale, float lambda, float eps, float out_scale,
                                         int* status, void* stream) {
    if (n_tiles <= 0) return 0;
    if (!pe_attention_diff_tcgen05_takes(H, G, D, Dv) || n_tiles > 65535 || q_stride % 8 || out_ld % 8 || out_col % 8 || !(scale > 0.f) || !status) return PE_ERR_UNSUPPORTED;
    if (((uintptr_t)q | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)out | (uintptr_t)tiles) & 15) return PE_ERR_UNSUPPORTED;
    if (pool_pages * 2 * G * DT_KTILE > 0x7fffff00ll) return PE_ERR_UNSUPPORTED;     // TMA coordinates are 32-bit
    CUtensorMap mq, mk, mv;
    int rc = at_make_map(&mq, q, n_tokens, (long long)2 * H * D, q_stride, DT_QTILE);
    if (rc) return rc;
    rc = at_make_map(&mk, k_pool, pool_pages * 2 * G * DT_KTILE, D, D, DT_KTILE);
    if (rc) return rc;
    rc = at_make_map(&mv, v_pool, pool_pages * G * DT_KTILE, Dv, Dv, DT_KTILE);
    if (rc) return rc;
    DtArgs p = {(bf16*)out, out_ld, out_col, table, table_stride, (const int4*)tiles, H, G, D, Dv, window, scale * 1.4426950408889634f, lambda, eps,
                out_scale, (int)(pool_pages * 2 * G * DT_KTILE), (int)(pool_pages * G * DT_KTILE)};
    cudaStream_t s = (cudaStream_t)stream;
    if (Dv <= 64) {
        PE_TRY(cudaFuncSetAttribute(attention_diff_tcgen05_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DT_SMEM_BYTES(1)));
        PE_TRY(pe_launch(attention_diff_tcgen05_kernel<1>, dim3(H, n_tiles), DT_THREADS, DT_SMEM_BYTES(1), s, mq, mk, mv, p, status));
    } else {
        PE_TRY(cudaFuncSetAttribute(attention_diff_tcgen05_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)DT_SMEM_BYTES(2)));
        PE_TRY(pe_launch(attention_diff_tcgen05_kernel<2>, dim3(H, n_tiles), DT_THREADS, DT_SMEM_BYTES(2), s, mq, mk, mv, p, status));
    }
    PE_LAUNCH_CHECK();
    return 0;
}

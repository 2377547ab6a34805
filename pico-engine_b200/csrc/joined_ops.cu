// Kernels around sublayers that read the same normed rows and share their first and last product, and around attention heads with
// several maps:
//  * heads_norm_store: on the rows of the first product, an RMS norm of every query and key row over its entries (one weight vector
//    for all query rows, one for all key rows), rotation in the layout of halves, and the cache write; there may be fewer value heads
//    than key heads (key heads that share values).
//  * map_difference: a head's output from the float32 outputs of its two maps, (a1 - lambda a2) divided by its root mean square.
//  * side_act: a feed-forward's activation from its columns of the first product into its columns of the last product's rows.
//  * route_rows: router product, softmax over all outputs, choice by score + correction, weights, from rows that are normed already.
#include "activations.cuh"

extern "C" void pe_set_pdl(int on) { pe_pdl_enabled() = on ? 1 : 0; }     // (this library's own copy of the switch)

// ---------------------------------------------------------------- norm, rotation and cache write of query and key rows
#define HN_THREADS 256
#define HN_MAX_D 256

struct HeadsNormArgs {
    void* proj; int ld, H, G, Gv, D, Dv;                          // a row begins with H*D query, G*D key and Gv*Dv value entries
    const void* q_w; int qw_dtype; const void* k_w; int kw_dtype; float eps;   // [D] each (null: that side is not normed)
    const float* freq; int rot;                                   // [rot / 2]; entry i < rot/2 turns with entry i + rot/2
    const int* tok_pos; const int* tok_row;
    void* k_pool; void* v_pool; const int* table; int table_stride; int store;
};

__device__ __forceinline__ int hn_pow2(int v) { int p = 1; while (p < v) p <<= 1; return p; }

// eight neighbouring entries of a norm weight (or ones)
__device__ __forceinline__ void hn_weights8(const void* w, int dtype, int at, float* f) {
    if (!w) {
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = 1.f;
    } else if (dtype == PE_BF16 && !((uintptr_t)w & 15)) {
        const uint4 r = *reinterpret_cast<const uint4*>((const bf16*)w + at);
        const __nv_bfloat162* r2 = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
        for (int e = 0; e < 4; ++e) { const float2 v = __bfloat1622float2(r2[e]); f[2 * e] = v.x; f[2 * e + 1] = v.y; }
    } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = load_as_f(w, dtype, at + e);
    }
}

// VEC: bfloat16 with D, Dv and the row length multiples of 8: a head is D / 8 neighbouring lanes (padded to a power of two), a lane
// holds eight entries; else a head is a warp and a lane holds every 32nd entry.  Normed rows meet in shared memory as float32 for the
// rotation.  A block a token (VEC: or gridDim.y blocks, each with its share of the heads, where the tokens are few); a pass's entries are
// asked for before the pass in front of it, and the first one's before the angles, are worked out.
template <typename T, bool VEC>
__global__ void __launch_bounds__(HN_THREADS) heads_norm_store_kernel(HeadsNormArgs a) {
    pdl_launch_dependents();
    __shared__ float s_cos[HN_MAX_D / 2], s_sin[HN_MAX_D / 2];
    __shared__ __align__(16) float s_row[HN_THREADS / 32][8 * 32];
    const int nt = blockDim.x, t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int D = a.D, half = a.rot >> 1, n_heads = a.H + a.G;
    T* row = (T*)a.proj + (size_t)t * a.ld;
    T* k_pool = (T*)a.k_pool;
    T* v_pool = (T*)a.v_pool;
    if constexpr (VEC) {
        const int L = D / 8, P = hn_pow2(L), per_warp = 32 / P;
        const int sub = lane / P, l = lane % P;
        const bool on = l < L;
        float* buf = s_row[warp] + sub * (P * 8);
        float qw[8], kw[8];
        if (on) { hn_weights8(a.q_w, a.qw_dtype, l * 8, qw); hn_weights8(a.k_w, a.kw_dtype, l * 8, kw); }
        pdl_wait();
        const int step = (nt / 32) * per_warp * gridDim.y;
        int h = (blockIdx.y * (nt / 32) + warp) * per_warp + sub;
        uint4 raw = make_uint4(0u, 0u, 0u, 0u);
        if (on && h < n_heads) raw = *reinterpret_cast<const uint4*>(row + (size_t)h * D + l * 8);
        const int pos = a.tok_pos[t], in_page = pos % PE_PAGE;
        long long page = -1;
        if (a.store) page = a.table[(size_t)a.tok_row[t] * a.table_stride + pos / PE_PAGE];
        for (int i = tid; i < half; i += nt) sincosf((float)pos * a.freq[i], &s_sin[i], &s_cos[i]);
        if (page >= 0) {
            const int per = a.Dv / 8;
            const T* v = row + (size_t)n_heads * D;
            for (int i = tid + blockIdx.y * nt; i < a.Gv * per; i += nt * gridDim.y) {
                const int c = i / per, d = (i % per) * 8;
                *reinterpret_cast<uint4*>(v_pool + (((size_t)page * a.Gv + c) * PE_PAGE + in_page) * a.Dv + d) = *reinterpret_cast<const uint4*>(v + (size_t)i * 8);
            }
        }
        __syncthreads();
        for (int h_first = h - sub; h_first < n_heads; h_first += step, h += step) {      // (the whole warp together)
            const bool live = on && h < n_heads;
            uint4 next = make_uint4(0u, 0u, 0u, 0u);
            if (on && h + step < n_heads) next = *reinterpret_cast<const uint4*>(row + (size_t)(h + step) * D + l * 8);
            float f[8];
            const __nv_bfloat162* r2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float2 v = __bfloat1622float2(r2[e]);
                f[2 * e] = v.x; f[2 * e + 1] = v.y;
                ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss);
            }
            for (int o = P >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const bool query = h < a.H;
            if (live && (query ? a.q_w : a.k_w)) {
                const float rstd = 1.0f / sqrtf(ss / (float)D + a.eps);
#pragma unroll
                for (int e = 0; e < 8; ++e) f[e] *= rstd * (query ? qw[e] : kw[e]);
            }
            if (half) {
                __syncwarp();
                if (live) {
                    *reinterpret_cast<float4*>(buf + l * 8) = make_float4(f[0], f[1], f[2], f[3]);
                    *reinterpret_cast<float4*>(buf + l * 8 + 4) = make_float4(f[4], f[5], f[6], f[7]);
                }
                __syncwarp();
                if (live && l * 8 < a.rot) {
#pragma unroll
                    for (int e = 0; e < 8; ++e) {
                        const int d = l * 8 + e;
                        if (d < half) f[e] = f[e] * s_cos[d] - buf[d + half] * s_sin[d];
                        else if (d < a.rot) f[e] = f[e] * s_cos[d - half] + buf[d - half] * s_sin[d - half];
                    }
                }
            }
            if (live) {
                __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
                for (int e = 0; e < 4; ++e) o2[e] = __floats2bfloat162_rn(f[2 * e], f[2 * e + 1]);
                if (query) *reinterpret_cast<uint4*>(row + (size_t)h * D + l * 8) = raw;
                else if (page >= 0) *reinterpret_cast<uint4*>(k_pool + (((size_t)page * a.G + (h - a.H)) * PE_PAGE + in_page) * D + l * 8) = raw;
            }
            raw = next;
        }
        return;
    }
    pdl_wait();
    const int pos = a.tok_pos[t], in_page = pos % PE_PAGE;
    long long page = -1;
    if (a.store) page = a.table[(size_t)a.tok_row[t] * a.table_stride + pos / PE_PAGE];
    for (int i = tid; i < half; i += nt) sincosf((float)pos * a.freq[i], &s_sin[i], &s_cos[i]);
    __syncthreads();
    float* buf = s_row[warp];
    for (int h = warp; h < n_heads; h += nt / 32) {
        T* v = row + (size_t)h * D;
        const void* w = h < a.H ? a.q_w : a.k_w;
        const int wd = h < a.H ? a.qw_dtype : a.kw_dtype;
        float ss = 0.f;
        for (int d = lane; d < D; d += 32) { const float x = to_f(v[d]); ss = fmaf(x, x, ss); }
        const float rstd = w ? 1.0f / sqrtf(warp_sum(ss) / (float)D + a.eps) : 1.f;
        __syncwarp();
        for (int d = lane; d < D; d += 32) buf[d] = w ? to_f(v[d]) * rstd * load_as_f(w, wd, d) : to_f(v[d]);
        __syncwarp();
        T* dst = h < a.H ? v : (page >= 0 ? k_pool + (((size_t)page * a.G + (h - a.H)) * PE_PAGE + in_page) * D : nullptr);
        if (dst) {
            for (int d = lane; d < D; d += 32) {
                float x = buf[d];
                if (d < half) x = x * s_cos[d] - buf[d + half] * s_sin[d];
                else if (d < a.rot) x = x * s_cos[d - half] + buf[d - half] * s_sin[d - half];
                dst[d] = from_f<T>(x);
            }
        }
    }
    if (page >= 0) {
        const T* v = row + (size_t)n_heads * D;
        for (int i = tid; i < a.Gv * a.Dv; i += nt) {
            const int c = i / a.Dv, d = i % a.Dv;
            v_pool[(((size_t)page * a.Gv + c) * PE_PAGE + in_page) * a.Dv + d] = v[i];
        }
    }
}

extern "C" int pe_heads_norm_store(void* proj, int dtype, int ld, int T, int H, int G, int Gv, int D, int Dv, const void* q_w, int qw_dtype,
                                   const void* k_w, int kw_dtype, float eps, const float* freq, int rot, const int* tok_pos,
                                   const int* tok_row, void* k_pool, void* v_pool, const int* table, int table_stride, int store, void* stream) {
    if (T <= 0) return 0;
    if (H <= 0 || G <= 0 || Gv <= 0 || D <= 0 || D > HN_MAX_D || Dv <= 0 || rot < 0 || rot > D || rot % 2 || ld < (H + G) * D + Gv * Dv) return PE_ERR_UNSUPPORTED;
    HeadsNormArgs a = {proj, ld, H, G, Gv, D, Dv, q_w, qw_dtype, k_w, kw_dtype, eps, freq, rot, tok_pos, tok_row, k_pool, v_pool, table, table_stride, store};
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = dtype == PE_BF16 && D % 8 == 0 && Dv % 8 == 0 && ld % 8 == 0 && !(((uintptr_t)proj | (uintptr_t)k_pool | (uintptr_t)v_pool) & 15);
    // many tokens: blocks of four warps; few: eight warps and as many blocks a token as its heads take passes
    int p = 1;
    while (p < D / 8) p <<= 1;
    const int per_pass = (HN_THREADS / 32) * (32 / p), passes = (H + G + per_pass - 1) / per_pass;
    const bool few = T * passes <= 4 * 148;
    if (dtype == PE_F32) PE_TRY(pe_launch(heads_norm_store_kernel<float, false>, T, HN_THREADS, 0, s, a));
    else if (dtype != PE_BF16) return PE_ERR_UNSUPPORTED;
    else if (vec) PE_TRY(pe_launch(heads_norm_store_kernel<bf16, true>, dim3(T, few ? passes : 1), few ? HN_THREADS : 128, 0, s, a));
    else PE_TRY(pe_launch(heads_norm_store_kernel<bf16, false>, T, HN_THREADS, 0, s, a));
    PE_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------- the difference of two maps
// maps [T][G][2][R][Dv] float32 (the outputs of the two maps of the R heads that share a key/value head); head h = g * R + r of token t:
// d = maps[t][g][0][r] - lambda * maps[t][g][1][r], out[t * out_ld + out_col + h * Dv ..] = d / sqrt(mean(d^2) + eps) * scale.  A warp a head.
template <typename T>
__global__ void __launch_bounds__(256) map_difference_kernel(const float* maps, int H, int R, int Dv, float lambda, float eps, float scale,
                                                             T* out, int out_ld, int out_col, size_t units) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t u = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (u >= units) return;
    const int lane = threadIdx.x & 31;
    const size_t t = u / H;
    const int h = (int)(u % H), g = h / R, r = h % R;
    const float* a1 = maps + ((t * (H / R) + g) * 2 * R + r) * Dv;
    const float* a2 = a1 + (size_t)R * Dv;
    float ss = 0.f;
    for (int d = lane; d < Dv; d += 32) { const float x = a1[d] - lambda * a2[d]; ss = fmaf(x, x, ss); }
    const float rstd = 1.0f / sqrtf(warp_sum(ss) / (float)Dv + eps) * scale;
    T* o = out + t * out_ld + out_col + (size_t)h * Dv;
    for (int d = lane; d < Dv; d += 32) o[d] = from_f<T>((a1[d] - lambda * a2[d]) * rstd);
}

extern "C" int pe_map_difference(const float* maps, int T, int H, int G, int Dv, float lambda, float eps, float scale, void* out, int dtype,
                                 int out_ld, int out_col, void* stream) {
    if (T <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || Dv <= 0 || out_ld < out_col + H * Dv || out_col < 0) return PE_ERR_UNSUPPORTED;
    const size_t units = (size_t)T * H;
    const unsigned blocks = (unsigned)((units + 7) / 8);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == PE_F32) PE_TRY(pe_launch(map_difference_kernel<float>, blocks, 256, 0, s, maps, H, H / G, Dv, lambda, eps, scale, (float*)out, out_ld, out_col, units));
    else if (dtype == PE_BF16) PE_TRY(pe_launch(map_difference_kernel<bf16>, blocks, 256, 0, s, maps, H, H / G, Dv, lambda, eps, scale, (bf16*)out, out_ld, out_col, units));
    else return PE_ERR_UNSUPPORTED;
    PE_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------- activations from columns of one matrix into columns of another
// out[t * out_ld + out_col + c] = act(in[t * ld + gate_col + c]) * in[t * ld + up_col + c] * colw[t * colw_ld + min(c / group, n_groups - 1)]
// for c < I, formed in float32 (up_col < 0: no second factor; colw null: no weights; a zero weight gives an exact zero).
__device__ __forceinline__ float side_act_of(float v, int act) { return act == 4 ? (v > 0.f ? v * v : 0.f) : go_act_fast(v, act); }

template <typename T>
__global__ void __launch_bounds__(256) side_act_kernel(const T* in, int ld, int gate_col, int up_col, int I, int act, const float* colw, int colw_ld,
                                                       int group, int n_groups, T* out, int out_ld, int out_col, size_t total) {
    pdl_launch_dependents();
    pdl_wait();
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
        const size_t t = idx / I;
        const int c = (int)(idx - t * I);
        const float w = colw ? colw[t * colw_ld + min(c / group, n_groups - 1)] : 1.f;
        float f = 0.f;
        if (w != 0.f) {
            f = go_act(to_f(in[t * ld + gate_col + c]), act) * w;
            if (up_col >= 0) f *= to_f(in[t * ld + up_col + c]);
        }
        out[t * out_ld + out_col + c] = from_f<T>(f);
    }
}

// bfloat16 with every column, row length and group a multiple of 8: eight columns of one group a thread with 16-byte accesses; hidden
// units whose weight is zero are not read.
__global__ void __launch_bounds__(256) side_act_vec_kernel(const bf16* in, int ld, int gate_col, int up_col, int I8, int act, const float* colw,
                                                           int colw_ld, int group8, int n_groups, bf16* out, int out_ld, int out_col, size_t total8) {
    pdl_launch_dependents();
    pdl_wait();
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total8; idx += (size_t)gridDim.x * blockDim.x) {
        const size_t t = idx / I8;
        const int c8 = (int)(idx - t * I8);
        const float w = colw ? colw[t * colw_ld + min(c8 / group8, n_groups - 1)] : 1.f;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (w != 0.f) {
            const bf16* row = in + t * ld + c8 * 8;
            v = *reinterpret_cast<const uint4*>(row + gate_col);
            uint4 u = make_uint4(0u, 0u, 0u, 0u);
            if (up_col >= 0) u = *reinterpret_cast<const uint4*>(row + up_col);
            __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&v);
            const __nv_bfloat162* q = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                float2 f = __bfloat1622float2(p[k]);
                f.x = side_act_of(f.x, act) * w; f.y = side_act_of(f.y, act) * w;
                if (up_col >= 0) { const float2 g = __bfloat1622float2(q[k]); f.x *= g.x; f.y *= g.y; }
                p[k] = __floats2bfloat162_rn(f.x, f.y);
            }
        }
        *reinterpret_cast<uint4*>(out + t * out_ld + out_col + c8 * 8) = v;
    }
}

extern "C" int pe_side_act(const void* in, int dtype, int ld, int gate_col, int up_col, int T, int I, int act, const float* colw, int colw_ld,
                           int group, int n_groups, void* out, int out_ld, int out_col, void* stream) {
    if (T <= 0 || I <= 0) return 0;
    if (gate_col < 0 || gate_col + I > ld || up_col + I > ld || out_col < 0 || out_col + I > out_ld || act == 5 || (colw && (group <= 0 || n_groups <= 0)))
        return PE_ERR_UNSUPPORTED;
    const size_t total = (size_t)T * I;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = dtype == PE_BF16 && I % 8 == 0 && ld % 8 == 0 && gate_col % 8 == 0 && (up_col < 0 || up_col % 8 == 0) && out_ld % 8 == 0 &&
                     out_col % 8 == 0 && (!colw || group % 8 == 0) && !(((uintptr_t)in | (uintptr_t)out) & 15);
    const size_t units = vec ? total / 8 : total;
    const int blocks = (int)((units + 255) / 256 < 148 * 16 ? (units + 255) / 256 : 148 * 16);
    if (vec) PE_TRY(pe_launch(side_act_vec_kernel, blocks, 256, 0, s, (const bf16*)in, ld, gate_col, up_col, I / 8, act, colw, colw_ld, colw ? group / 8 : 1,
                              n_groups, (bf16*)out, out_ld, out_col, units));
    else if (dtype == PE_F32) PE_TRY(pe_launch(side_act_kernel<float>, blocks, 256, 0, s, (const float*)in, ld, gate_col, up_col, I, act, colw, colw_ld, group,
                                               n_groups, (float*)out, out_ld, out_col, total));
    else if (dtype == PE_BF16) PE_TRY(pe_launch(side_act_kernel<bf16>, blocks, 256, 0, s, (const bf16*)in, ld, gate_col, up_col, I, act, colw, colw_ld, group,
                                                n_groups, (bf16*)out, out_ld, out_col, total));
    else return PE_ERR_UNSUPPORTED;
    PE_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------- the router over all experts, with a correction of the choice
// Rows h [T, K] (float32 or bfloat16), router [n, K] in the rows' dtype, n = N + (gate ? 1 : 0) rows: logits z = router . h with float32 sums.
// Scores s = softmax over the first N logits; the choice reads s + correction [N] (null: s), the `top` largest win (of equal numbers the
// lower index first); their weights are factor * s.  out [T, E + gate + (N > E)] float32, E <= N: the weights of experts 0 .. E-1 (zero
// where not chosen), then sigmoid(logit N) where there is a gate, then the sum of the weights of the chosen among E .. N-1 (experts
// whose output is their input).  ids [T, top] (or null): the chosen, largest choice score first.
#define RR_THREADS 256
#define RR_WARPS 8
#define RR_MAX_N 1024

__device__ __forceinline__ void rr_choose(float* z, int N, int E, int gate, const void* corr, int corr_dtype, int top, float factor, float* w,
                                          int* ids, int lane) {
    float m = -INFINITY;
    for (int e = lane; e < N; e += 32) m = fmaxf(m, z[e]);
    m = warp_max(m);
    float all = 0.f;
    for (int e = lane; e < N; e += 32) all += expf(z[e] - m);
    const float inv = 1.0f / warp_sum(all);
    const int cols = E + gate;
    for (int e = lane; e < E; e += 32) w[e] = 0.f;
    if (gate && lane == 0) w[E] = go_sigmoid(z[N]);
    __syncwarp();
    unsigned taken = 0u;                                       // the lane's taken places (a lane sees N / 32 <= 32 of them)
    float passed = 0.f;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int at = 0x7fffffff;
        for (int e = lane, i = 0; e < N; e += 32, ++i) {
            if (taken >> i & 1u) continue;
            const float c = expf(z[e] - m) * inv + (corr ? load_as_f(corr, corr_dtype, e) : 0.f);
            if (c > best || (c == best && e < at) || at == 0x7fffffff) { best = c; at = e; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, at, o);
            if (oa != 0x7fffffff && (at == 0x7fffffff || ob > best || (ob == best && oa < at))) { best = ob; at = oa; }
        }
        if (at == 0x7fffffff) break;
        if ((at & 31) == lane) taken |= 1u << (at >> 5);
        const float s = factor * (expf(z[at] - m) * inv);
        if (at >= E) passed += s;
        else if (lane == 0) w[at] = s;
        if (lane == 0 && ids) ids[k] = at;
    }
    if (N > E && lane == 0) w[cols] = passed;
}

__device__ __forceinline__ void rr_load8(const float* p, float* f) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void rr_load8(const bf16* p, float* f) {
    const uint4 r = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* r2 = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
    for (int e = 0; e < 4; ++e) { const float2 v = __bfloat1622float2(r2[e]); f[2 * e] = v.x; f[2 * e + 1] = v.y; }
}

// A block takes TB tokens, whose rows it keeps in shared memory; a warp takes two rows of the router at a time for all of them, its
// lanes eight columns each (VEC) or one, so that a row of the router is read once for TB tokens; a token's logit is the same sum in the
// same order whatever TB is.  Then a warp a token chooses.
template <typename T, int TB, bool VEC>
__global__ void __launch_bounds__(RR_THREADS) route_rows_kernel(const T* h, const T* router, int K, int N, int E, int gate, const void* corr,
                                                                int corr_dtype, int top, float factor, float* out, int* ids, int n_tokens) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char rr_smem[];
    T* rows = reinterpret_cast<T*>(rr_smem);                  // [TB][K]
    __shared__ float z[TB][RR_MAX_N + 1];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int t0 = blockIdx.x * TB, nt = min(TB, n_tokens - t0), n = N + gate;
    pdl_wait();
    if constexpr (VEC) {
        constexpr int PER = 16 / (int)sizeof(T);
        const uint4* src = reinterpret_cast<const uint4*>(h + (size_t)t0 * K);
        for (int i = tid; i < TB * K / PER; i += RR_THREADS)
            reinterpret_cast<uint4*>(rows)[i] = i < nt * K / PER ? src[i] : make_uint4(0u, 0u, 0u, 0u);
    } else {
        for (int i = tid; i < TB * K; i += RR_THREADS) rows[i] = i < nt * K ? h[(size_t)t0 * K + i] : from_f<T>(0.f);
    }
    __syncthreads();
    for (int e0 = warp * 2; e0 < n; e0 += 2 * RR_WARPS) {
        const T* r0 = router + (size_t)e0 * K;
        const T* r1 = e0 + 1 < n ? r0 + K : r0;
        float acc[2][TB];
#pragma unroll
        for (int b = 0; b < TB; ++b) acc[0][b] = acc[1][b] = 0.f;
        if constexpr (VEC) {
#pragma unroll 2
            for (int k = lane * 8; k < K; k += 256) {
                float w0[8], w1[8];
                rr_load8(r0 + k, w0);
                rr_load8(r1 + k, w1);
#pragma unroll
                for (int b = 0; b < TB; ++b) {
                    float x[8];
                    rr_load8(rows + (size_t)b * K + k, x);
#pragma unroll
                    for (int j = 0; j < 8; ++j) { acc[0][b] = fmaf(x[j], w0[j], acc[0][b]); acc[1][b] = fmaf(x[j], w1[j], acc[1][b]); }
                }
            }
        } else {
            for (int k = lane; k < K; k += 32) {
                const float w0 = to_f(r0[k]), w1 = to_f(r1[k]);
#pragma unroll
                for (int b = 0; b < TB; ++b) {
                    const float x = to_f(rows[(size_t)b * K + k]);
                    acc[0][b] = fmaf(x, w0, acc[0][b]); acc[1][b] = fmaf(x, w1, acc[1][b]);
                }
            }
        }
#pragma unroll
        for (int b = 0; b < TB; ++b) {
            const float s0 = warp_sum(acc[0][b]), s1 = warp_sum(acc[1][b]);
            if (lane == 0) { z[b][e0] = s0; if (e0 + 1 < n) z[b][e0 + 1] = s1; }
        }
    }
    __syncthreads();
    const int cols = E + gate + (N > E ? 1 : 0);
    for (int b = warp; b < nt; b += RR_WARPS)
        rr_choose(z[b], N, E, gate, corr, corr_dtype, top, factor, out + (size_t)(t0 + b) * cols, ids ? ids + (size_t)(t0 + b) * top : nullptr, lane);
}

template <typename T, int TB>
static int rr_launch(const void* h, const void* router, int K, int N, int E, int gate, const void* corr, int corr_dtype, int top, float factor,
                     float* out, int* ids, int n_tokens, cudaStream_t s) {
    const size_t smem = sizeof(T) * (size_t)TB * K;
    const bool vec = K % 8 == 0 && !(((uintptr_t)h | (uintptr_t)router) & 15);
    if (vec) {
        PE_TRY(cudaFuncSetAttribute(route_rows_kernel<T, TB, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        PE_TRY(pe_launch(route_rows_kernel<T, TB, true>, (n_tokens + TB - 1) / TB, RR_THREADS, smem, s, (const T*)h, (const T*)router, K, N, E, gate, corr,
                         corr_dtype, top, factor, out, ids, n_tokens));
    } else {
        PE_TRY(cudaFuncSetAttribute(route_rows_kernel<T, TB, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        PE_TRY(pe_launch(route_rows_kernel<T, TB, false>, (n_tokens + TB - 1) / TB, RR_THREADS, smem, s, (const T*)h, (const T*)router, K, N, E, gate, corr,
                         corr_dtype, top, factor, out, ids, n_tokens));
    }
    PE_LAUNCH_CHECK();
    return 0;
}

extern "C" int pe_route_rows(const void* h, int dtype, const void* router, int K, int N, int E, int gate, const void* corr, int corr_dtype, int top,
                             float factor, float* out, int* ids, int T, void* stream) {
    if (T <= 0) return 0;
    if (K <= 0 || N <= 0 || N > RR_MAX_N || E < 0 || E > N || top <= 0 || top > N || gate < 0 || gate > 1 || (dtype != PE_F32 && dtype != PE_BF16))
        return PE_ERR_UNSUPPORTED;
    const size_t row = (size_t)K * (dtype == PE_F32 ? 4 : 2);
    if (row > 180 * 1024) return PE_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const bool many = T >= 4 * 148 && 4 * row <= 96 * 1024;
    if (dtype == PE_F32) return many ? rr_launch<float, 4>(h, router, K, N, E, gate, corr, corr_dtype, top, factor, out, ids, T, s)
                                     : rr_launch<float, 1>(h, router, K, N, E, gate, corr, corr_dtype, top, factor, out, ids, T, s);
    return many ? rr_launch<bf16, 4>(h, router, K, N, E, gate, corr, corr_dtype, top, factor, out, ids, T, s)
                : rr_launch<bf16, 1>(h, router, K, N, E, gate, corr, corr_dtype, top, factor, out, ids, T, s);
}

// Kernels around two mixers that stand side by side and share their first and last product, and around a residual of several
// streams:
//  * heads_prepare: on the rows of the shared first product, (job 0) an RMS norm over all query entries of a token at once and one
//    over all its key entries, rotation, and the cache write of an attention; (job 1) rotation and scale of the queries and keys of
//    a linear attention, written as float32 rows of their own.  One launch does both jobs.
//  * gate_heads: the mixers' outputs, normed a run of channels at a time or not, times an activation of a gate, times the mixer's
//    weight, side by side as the rows the shared last product reads.  One launch does all mixers.
//  * stream_mix: the streams after a sublayer (a small matrix times the streams, plus the sublayer's output times a number a stream),
//    and in the same pass what the next sublayer reads (a weighted sum of the new streams, RMS-normed).
#include "activations.cuh"

// ---------------------------------------------------------------- rotations
// A head of D entries with the first `rot` turned is D - rot/2 units: unit u < rot/2 is the pair (a, b) of that index, in the layout
// of neighbours (2u, 2u + 1) or of halves (u, u + rot/2); the others are single entries.  A thread that owns a unit reads and writes
// its entries alone, so rows can be rewritten in place.
__device__ __forceinline__ void bo_unit(int u, int rot, int halves, int& a, int& b) {
    const int half = rot >> 1;
    if (u >= half) { a = rot + (u - half); b = -1; return; }
    if (halves) { a = u; b = u + half; } else { a = 2 * u; b = 2 * u + 1; }
}

struct HeadsArgs {
    void* proj; int ld, T;
    const int* tok_pos; const int* tok_row;
    // job 0: attention (H = 0: there is none)
    int H, G, D, Dv;
    const void* q_w; const void* k_w; int w_dtype; float eps;      // norm weights over H*D and G*D entries (null: no norm)
    const float* freq; int rot, halves;
    void* k_pool; void* v_pool; const int* table; int table_stride; int store;
    // job 1: linear attention (RH = 0: there is none)
    int RH, RD, r_q, r_k;                                          // heads, head size, first columns of queries and keys
    const float* r_freq; int r_rot, r_halves; float k_scale;
    float* r_out;                                                  // [T, 2 * RH * RD]: queries | keys
};

// Two block-wide sums at once, the same values returned to every thread.
__device__ __forceinline__ float2 bo_block_sum2(float a, float b, float2* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    a = warp_sum(a); b = warp_sum(b);
    if (lane == 0) scratch[warp] = make_float2(a, b);
    __syncthreads();
    float2 t = lane < nwarps ? scratch[lane] : make_float2(0.f, 0.f);
    return make_float2(warp_sum(t.x), warp_sum(t.y));
}

// VEC (bfloat16, neighbours, D and rot multiples of 8, up to 8192 query and key entries, aligned rows and weights in bfloat16): a
// thread keeps up to four runs of eight entries in registers between the sums of squares and the rotation.
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) heads_prepare_kernel(HeadsArgs a) {
    pdl_launch_dependents();
    __shared__ float s_cos[128], s_sin[128];
    __shared__ float2 red[8];
    pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
    const int job = blockIdx.y + (a.H > 0 ? 0 : 1);
    T* row = (T*)a.proj + (size_t)t * a.ld;
    const int pos = a.tok_pos[t];
    // the row's entries are asked for before the angles are worked out
    uint4 raw[VEC ? 4 : 1];
    if constexpr (VEC) {
        if (job == 0) {
            const int units = (a.H + a.G) * a.D / 8;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = tid + e * nt;
                raw[e] = i < units ? *reinterpret_cast<const uint4*>(row + i * 8) : make_uint4(0u, 0u, 0u, 0u);
            }
        }
    }
    long long page = -1;
    if (job == 0 && a.store) page = a.table[(size_t)a.tok_row[t] * a.table_stride + pos / PE_PAGE];
    const float* freq = job == 0 ? a.freq : a.r_freq;
    const int half = (job == 0 ? a.rot : a.r_rot) / 2;
    for (int i = tid; i < half; i += nt) sincosf((float)pos * freq[i], &s_sin[i], &s_cos[i]);
    if (job == 1) {
        __syncthreads();
        const int D = a.RD, rot = a.r_rot, n = a.RH * D;
        float* out = a.r_out + (size_t)t * 2 * n;
        if (sizeof(T) == 2 && a.r_halves && half % 2 == 0 && D % 2 == 0 && a.r_q % 2 == 0 && a.r_k % 2 == 0 && a.ld % 2 == 0) {
            // two neighbouring pairs (or two neighbouring single entries) a thread: 4-byte reads, 8-byte writes
            const int per = (D - half) / 2, units = 2 * a.RH * per;
#pragma unroll 2
            for (int i = tid; i < units; i += nt) {
                const int h = i / per, u = 2 * (i - h * per);
                const bool key = h >= a.RH;
                const T* src = row + (key ? a.r_k + (h - a.RH) * D : a.r_q + h * D);
                float* dst = out + (size_t)h * D;
                const float s = key ? a.k_scale : 1.f;
                const int e = u < half ? u : rot + (u - half);
                const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + e));
                if (u < half) {
                    const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(src + e + half));
                    const float c0 = s_cos[u], c1 = s_cos[u + 1], n0 = s_sin[u], n1 = s_sin[u + 1];
                    *reinterpret_cast<float2*>(dst + e) = make_float2(s * fmaf(x.x, c0, -y.x * n0), s * fmaf(x.y, c1, -y.y * n1));
                    *reinterpret_cast<float2*>(dst + e + half) = make_float2(s * fmaf(y.x, c0, x.x * n0), s * fmaf(y.y, c1, x.y * n1));
                } else *reinterpret_cast<float2*>(dst + e) = make_float2(s * x.x, s * x.y);
            }
            return;
        }
        const int per = D - half, units = 2 * a.RH * per;
        for (int i = tid; i < units; i += nt) {
            const int h = i / per, u = i - h * per;
            const bool key = h >= a.RH;
            const T* src = row + (key ? a.r_k + (h - a.RH) * D : a.r_q + h * D);
            float* dst = out + (size_t)h * D;
            const float s = key ? a.k_scale : 1.f;
            int e, p;
            bo_unit(u, rot, a.r_halves, e, p);
            const float x = to_f(src[e]);
            if (p >= 0) {
                const float y = to_f(src[p]);
                dst[e] = s * fmaf(x, s_cos[u], -y * s_sin[u]);
                dst[p] = s * fmaf(y, s_cos[u], x * s_sin[u]);
            } else dst[e] = s * x;
        }
        return;
    }
    const int D = a.D, nq = a.H * D, nk = a.G * D;
    const int in_page = pos % PE_PAGE;
    T* k_pool = (T*)a.k_pool;
    T* v_pool = (T*)a.v_pool;
    const bool store = a.store && page >= 0;
    if constexpr (VEC) {
        float sq = 0.f, sk = 0.f;
        const int units = (nq + nk) / 8;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = tid + e * nt;
            const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw[e]);
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(p[j]); ss = fmaf(f.x, f.x, fmaf(f.y, f.y, ss)); }
            if (i * 8 < nq) sq += ss; else sk += ss;
        }
        const float2 sums = bo_block_sum2(sq, sk, red);                    // (its barrier also publishes the angles)
        const float rq = a.q_w ? 1.0f / sqrtf(sums.x / (float)nq + a.eps) : 1.f;
        const float rk = a.k_w ? 1.0f / sqrtf(sums.y / (float)nk + a.eps) : 1.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = tid + e * nt;
            if (i >= units) break;
            const int at = i * 8, d = at % D;
            const bool key = at >= nq;
            const float r = key ? rk : rq;
            const void* w = key ? a.k_w : a.q_w;
            __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&raw[e]);
            uint4 wr = make_uint4(0u, 0u, 0u, 0u);
            if (w) wr = *reinterpret_cast<const uint4*>((const bf16*)w + (key ? at - nq : at));
            const __nv_bfloat162* wp = reinterpret_cast<const __nv_bfloat162*>(&wr);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float2 f = __bfloat1622float2(p[j]);
                f.x *= r; f.y *= r;
                if (w) { const float2 g = __bfloat1622float2(wp[j]); f.x *= g.x; f.y *= g.y; }
                if (d < a.rot) {
                    const float c = s_cos[d / 2 + j], n = s_sin[d / 2 + j];
                    f = make_float2(fmaf(f.x, c, -f.y * n), fmaf(f.y, c, f.x * n));
                }
                p[j] = __floats2bfloat162_rn(f.x, f.y);
            }
            *reinterpret_cast<uint4*>(row + at) = raw[e];
            if (key && store)
                *reinterpret_cast<uint4*>(k_pool + (((size_t)page * a.G + (at - nq) / D) * PE_PAGE + in_page) * D + d) = raw[e];
        }
        if (store) {
            const int Dv = a.Dv;
            if (Dv % 8 == 0) {
                for (int i = tid; i < a.G * Dv / 8; i += nt) {
                    const int c = i * 8 / Dv, d = i * 8 % Dv;
                    *reinterpret_cast<uint4*>(v_pool + (((size_t)page * a.G + c) * PE_PAGE + in_page) * Dv + d) =
                        *reinterpret_cast<const uint4*>(row + nq + nk + i * 8);
                }
            } else {
                for (int i = tid; i < a.G * Dv; i += nt)
                    v_pool[(((size_t)page * a.G + i / Dv) * PE_PAGE + in_page) * Dv + i % Dv] = row[nq + nk + i];
            }
        }
        return;
    }
    float sq = 0.f, sk = 0.f;
    for (int i = tid; i < nq + nk; i += nt) {
        const float f = to_f(row[i]);
        if (i < nq) sq = fmaf(f, f, sq); else sk = fmaf(f, f, sk);
    }
    const float2 sums = bo_block_sum2(sq, sk, red);
    const float rq = a.q_w ? 1.0f / sqrtf(sums.x / (float)nq + a.eps) : 1.f;
    const float rk = a.k_w ? 1.0f / sqrtf(sums.y / (float)nk + a.eps) : 1.f;
    const int per = D - half, units = (a.H + a.G) * per;
    for (int i = tid; i < units; i += nt) {
        const int h = i / per, u = i - h * per;
        const bool key = h >= a.H;
        const float r = key ? rk : rq;
        const void* w = key ? a.k_w : a.q_w;
        const int base = key ? (h - a.H) * D : h * D;                      // within all queries or all keys
        int e, p;
        bo_unit(u, a.rot, a.halves, e, p);
        T* head = row + (size_t)h * D;
        T* dst = key && store ? k_pool + (((size_t)page * a.G + (h - a.H)) * PE_PAGE + in_page) * D : nullptr;
        float x = to_f(head[e]) * r;
        if (w) x *= load_as_f(w, a.w_dtype, base + e);
        if (p >= 0) {
            float y = to_f(head[p]) * r;
            if (w) y *= load_as_f(w, a.w_dtype, base + p);
            const float x1 = fmaf(x, s_cos[u], -y * s_sin[u]), y1 = fmaf(y, s_cos[u], x * s_sin[u]);
            const T yo = from_f<T>(y1);
            head[p] = yo;
            if (dst) dst[p] = yo;
            x = x1;
        }
        const T xo = from_f<T>(x);
        head[e] = xo;
        if (dst) dst[e] = xo;
    }
    if (store)
        for (int i = tid; i < a.G * a.Dv; i += nt)
            v_pool[(((size_t)page * a.G + i / a.Dv) * PE_PAGE + in_page) * a.Dv + i % a.Dv] = row[nq + nk + i];
}

extern "C" int pe_heads_prepare(void* proj, int dtype, int ld, int T, const int* tok_pos, const int* tok_row,
                                int H, int G, int D, int Dv, const void* q_w, const void* k_w, int w_dtype, float eps, const float* freq,
                                int rot, int halves, void* k_pool, void* v_pool, const int* table, int table_stride, int store,
                                int RH, int RD, int r_q, int r_k, const float* r_freq, int r_rot, int r_halves, float k_scale, float* r_out,
                                void* stream) {
    if (T <= 0) return 0;
    if (H < 0 || RH < 0 || (H == 0 && RH == 0)) return PE_ERR_UNSUPPORTED;
    if (H > 0 && (G <= 0 || D <= 0 || D > 256 || Dv <= 0 || rot < 0 || rot > D || (rot & 1) || (rot > 0 && !freq) || ld < (H + G) * D + G * Dv ||
                  (store && (!k_pool || !v_pool || !table)))) return PE_ERR_UNSUPPORTED;
    if (RH > 0 && (RD <= 0 || RD > 256 || r_rot < 0 || r_rot > RD || (r_rot & 1) || (r_rot > 0 && !r_freq) || !r_out || r_q < 0 || r_k < 0 ||
                   ld < r_q + RH * RD || ld < r_k + RH * RD || ((uintptr_t)r_out & 7))) return PE_ERR_UNSUPPORTED;
    HeadsArgs a = {proj, ld, T, tok_pos, tok_row, H, G, D, Dv, q_w, k_w, w_dtype, eps, freq, rot, halves, k_pool, v_pool, table, table_stride, store,
                   RH, RD, r_q, r_k, r_freq, r_rot, r_halves, k_scale, r_out};
    const dim3 grid(T, (H > 0) + (RH > 0));
    cudaStream_t s = (cudaStream_t)stream;
    const int widest = H > 0 ? (H + G) * D / 8 : RH * RD / 2;
    const int threads = widest > 128 ? 256 : 128;
    if (dtype == PE_BF16) {
        const bool vec = H > 0 && !halves && D % 8 == 0 && rot % 8 == 0 && ld % 8 == 0 && (H + G) * D <= 4 * 8 * threads && (w_dtype == PE_BF16 || (!q_w && !k_w)) &&
                         !(((uintptr_t)proj | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)q_w | (uintptr_t)k_w) & 15);
        if (vec) PE_TRY(pe_launch(heads_prepare_kernel<bf16, true>, grid, threads, 0, s, a));
        else PE_TRY(pe_launch(heads_prepare_kernel<bf16, false>, grid, threads, 0, s, a));
    } else if (dtype == PE_F32) PE_TRY(pe_launch(heads_prepare_kernel<float, false>, grid, threads, 0, s, a));
    else return PE_ERR_UNSUPPORTED;
    PE_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------- outputs of mixers times their gates, side by side
// Mixer j has rows in_j [T, C_j] (float32 or the step's dtype).  group_j > 0: every run of so many channels is divided by
// sqrt(mean(run^2) + eps_j) and multiplied by weight_j [group_j] (null: ones); then everything is multiplied by
// act_j(gate[t, gate_off_j + c]) and by scale_j and rounded once into out[t, out_off_j + c].  `pad` columns behind the last mixer's
// become zeros.  A block a (token, mixer).
struct GateJob { const void* in; int in_f32, C, group; const void* weight; int w_dtype; float eps; int gate_off, act; float scale; int out_off; };
struct GateArgs { GateJob job[4]; int n, gate_ld, out_ld, pad; const void* gate; void* out; };

template <typename T>
__device__ __forceinline__ float bo_act(float v, int act) { return sizeof(T) == 2 ? go_act_fast(v, act) : go_act(v, act); }

// Four channels at a time; every width and offset a multiple of 4.
__device__ __forceinline__ float4 bo_load4(const void* p, int f32, size_t i) {
    if (f32) return *reinterpret_cast<const float4*>((const float*)p + i);
    const uint2 r = *reinterpret_cast<const uint2*>((const bf16*)p + i);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void bo_gate4(const GateJob& j, const bf16* gate, bf16* out, float4 f, float r, int c, int in_run) {
    const float4 g = bo_load4(gate, 0, j.gate_off + c);
    r *= j.scale;
    f.x *= r * go_act_fast(g.x, j.act); f.y *= r * go_act_fast(g.y, j.act); f.z *= r * go_act_fast(g.z, j.act); f.w *= r * go_act_fast(g.w, j.act);
    if (j.weight) {
        f.x *= load_as_f(j.weight, j.w_dtype, in_run); f.y *= load_as_f(j.weight, j.w_dtype, in_run + 1);
        f.z *= load_as_f(j.weight, j.w_dtype, in_run + 2); f.w *= load_as_f(j.weight, j.w_dtype, in_run + 3);
    }
    uint2 o;
    *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(f.x, f.y);
    *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(f.z, f.w);
    *reinterpret_cast<uint2*>(out + j.out_off + c) = o;
}

__global__ void __launch_bounds__(256) gate_heads_x4_kernel(GateArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
    const GateJob& j = a.job[blockIdx.y];
    const bf16* gate = (const bf16*)a.gate + (size_t)t * a.gate_ld;
    bf16* out = (bf16*)a.out + (size_t)t * a.out_ld;
    const size_t in0 = (size_t)t * j.C;
    if (blockIdx.y == 0 && tid < a.pad) out[a.out_ld - a.pad + tid] = __float2bfloat16_rn(0.f);
    if (j.group == 0) {
        for (int i = tid; i < j.C / 4; i += blockDim.x) bo_gate4(j, gate, out, bo_load4(j.in, j.in_f32, in0 + 4 * i), 1.f, 4 * i, 0);
        return;
    }
    for (int run = warp; run < j.C / j.group; run += nw) {                 // a warp a run of up to 512 channels, kept in registers
        const int c0 = run * j.group, nv = j.group / 4;
        float4 v[4];
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = lane + 32 * e;
            v[e] = i < nv ? bo_load4(j.in, j.in_f32, in0 + c0 + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
            ss += v[e].x * v[e].x + v[e].y * v[e].y + v[e].z * v[e].z + v[e].w * v[e].w;
        }
        const float r = 1.0f / sqrtf(warp_sum(ss) / (float)j.group + j.eps);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = lane + 32 * e;
            if (i < nv) bo_gate4(j, gate, out, v[e], r, c0 + 4 * i, 4 * i);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) gate_heads_kernel(GateArgs a) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
    const GateJob& j = a.job[blockIdx.y];
    const T* gate = (const T*)a.gate + (size_t)t * a.gate_ld + j.gate_off;
    T* out = (T*)a.out + (size_t)t * a.out_ld;
    const size_t in0 = (size_t)t * j.C;
    if (blockIdx.y == 0)
        for (int i = tid; i < a.pad; i += blockDim.x) out[a.out_ld - a.pad + i] = from_f<T>(0.f);
    out += j.out_off;
    auto load = [&](int c) { return j.in_f32 ? ((const float*)j.in)[in0 + c] : to_f(((const T*)j.in)[in0 + c]); };
    if (j.group == 0) {
        for (int c = tid; c < j.C; c += blockDim.x) out[c] = from_f<T>(load(c) * bo_act<T>(to_f(gate[c]), j.act) * j.scale);
        return;
    }
    for (int run = warp; run < j.C / j.group; run += nw) {
        const int c0 = run * j.group;
        float ss = 0.f;
        for (int i = lane; i < j.group; i += 32) { const float f = load(c0 + i); ss = fmaf(f, f, ss); }
        const float r = 1.0f / sqrtf(warp_sum(ss) / (float)j.group + j.eps);
        for (int i = lane; i < j.group; i += 32) {
            float f = load(c0 + i) * r;
            if (j.weight) f *= load_as_f(j.weight, j.w_dtype, i);
            out[c0 + i] = from_f<T>(f * bo_act<T>(to_f(gate[c0 + i]), j.act) * j.scale);
        }
    }
}

// The jobs come as arrays of n entries (host memory).
extern "C" int pe_gate_heads(int n, const void* const* in, const int* in_f32, const int* C, const int* group, const void* const* weight,
                             const int* w_dtype, const float* eps, const int* gate_off, const int* act, const float* scale, const int* out_off,
                             int T, const void* gate, int gate_ld, void* out, int out_ld, int dtype, void* stream) {
    if (T <= 0) return 0;
    if (n < 1 || n > 4) return PE_ERR_UNSUPPORTED;
    GateArgs a = {};
    a.n = n; a.gate = gate; a.gate_ld = gate_ld; a.out = out; a.out_ld = out_ld;
    int end = 0, widest = 0;
    bool x4 = dtype == PE_BF16 && gate_ld % 4 == 0 && out_ld % 4 == 0 && !(((uintptr_t)gate | (uintptr_t)out) & 7);
    for (int i = 0; i < n; ++i) {
        if (C[i] <= 0 || group[i] < 0 || (group[i] > 0 && C[i] % group[i]) || gate_off[i] < 0 || gate_off[i] + C[i] > gate_ld || out_off[i] != end)
            return PE_ERR_UNSUPPORTED;
        a.job[i] = {in[i], in_f32[i] || dtype == PE_F32, C[i], group[i], weight[i], w_dtype[i], eps[i], gate_off[i], act[i], scale[i], out_off[i]};
        end += C[i];
        widest = C[i] > widest ? C[i] : widest;
        x4 = x4 && C[i] % 4 == 0 && gate_off[i] % 4 == 0 && out_off[i] % 4 == 0 && group[i] % 4 == 0 && group[i] <= 512 && !((uintptr_t)in[i] & (in_f32[i] ? 15 : 7));
        if (act[i] < 0 || act[i] == 5 || act[i] == 4) return PE_ERR_UNSUPPORTED;
    }
    a.pad = out_ld - end;
    if (a.pad < 0 || a.pad > 32) return PE_ERR_UNSUPPORTED;
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 grid(T, n);
    const int threads = widest > 512 ? 256 : 128;
    if (x4) PE_TRY(pe_launch(gate_heads_x4_kernel, grid, threads, 0, s, a));
    else if (dtype == PE_F32) PE_TRY(pe_launch(gate_heads_kernel<float>, grid, threads, 0, s, a));
    else if (dtype == PE_BF16) PE_TRY(pe_launch(gate_heads_kernel<bf16>, grid, threads, 0, s, a));
    else return PE_ERR_UNSUPPORTED;
    PE_LAUNCH_CHECK();
    return 0;
}

// ---------------------------------------------------------------- streams
// The residual is S streams x [T, S, W] float32.  With a pending sublayer output y [T, W]: x_t <- sum_s mix[s, t] x_s + out[t] y, all from
// the old ones, stored to dst (null: not stored).  Then, with h: u = sum_s in[s] x_s of the streams as they now stand (in null: their
// plain sum), and h = u / sqrt(mean(u^2) + eps) * weight (weight null: u itself), in h's dtype.  src may be one matrix that all streams
// still equal (src_stream = 0).  A thread reads all streams of its columns before it writes any, so dst may be src.
struct StreamArgs {
    const float* src; long long src_tok, src_stream;
    float* dst;
    const void* y; int y_dtype; const float* mix; const float* out;
    const float* in; const void* weight; int w_dtype; float eps;
    void* h;
    int S, W;
};

// Four columns a thread and step, up to four steps kept for the norm (W up to 4 * 4 * threads).
template <int S, typename TH>
__global__ void __launch_bounds__(256) stream_mix_x4_kernel(StreamArgs a) {
    pdl_launch_dependents();
    __shared__ float s_mix[S * S + 2 * S], red[33];
    const int tid = threadIdx.x, nt = blockDim.x;
    const bool pending = a.y != nullptr;
    for (int i = tid; i < S * S; i += nt) s_mix[i] = pending ? a.mix[i] : 0.f;         // weights: no kernel writes them
    for (int i = tid; i < S; i += nt) { s_mix[S * S + i] = pending ? a.out[i] : 0.f; s_mix[S * S + S + i] = a.in ? a.in[i] : 1.f; }
    __syncthreads();
    pdl_wait();
    const size_t t = blockIdx.x;
    const int nv = a.W / 4;
    float4 u[4];
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        u[e] = make_float4(0.f, 0.f, 0.f, 0.f);
        const int i = tid + e * nt;
        if (i < nv) {
            float4 x[S];
#pragma unroll
            for (int s = 0; s < S; ++s) x[s] = *reinterpret_cast<const float4*>(a.src + t * a.src_tok + s * a.src_stream + 4 * i);
            if (pending) {
                float4 y;
                if (a.y_dtype == PE_F32) y = *reinterpret_cast<const float4*>((const float*)a.y + t * a.W + 4 * i);
                else y = bo_load4(a.y, 0, t * a.W + 4 * i);
#pragma unroll
                for (int to = 0; to < S; ++to) {
                    const float o = s_mix[S * S + to];
                    float4 n = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
                    for (int s = 0; s < S; ++s) {
                        const float m = s_mix[s * S + to];
                        n.x = fmaf(m, x[s].x, n.x); n.y = fmaf(m, x[s].y, n.y); n.z = fmaf(m, x[s].z, n.z); n.w = fmaf(m, x[s].w, n.w);
                    }
                    if (a.dst) *reinterpret_cast<float4*>(a.dst + (t * S + to) * a.W + 4 * i) = n;
                    const float g = s_mix[S * S + S + to];
                    u[e].x = fmaf(g, n.x, u[e].x); u[e].y = fmaf(g, n.y, u[e].y); u[e].z = fmaf(g, n.z, u[e].z); u[e].w = fmaf(g, n.w, u[e].w);
                }
            } else {
#pragma unroll
                for (int s = 0; s < S; ++s) {
                    const float g = s_mix[S * S + S + s];
                    u[e].x = fmaf(g, x[s].x, u[e].x); u[e].y = fmaf(g, x[s].y, u[e].y); u[e].z = fmaf(g, x[s].z, u[e].z); u[e].w = fmaf(g, x[s].w, u[e].w);
                    if (a.dst) *reinterpret_cast<float4*>(a.dst + (t * S + s) * a.W + 4 * i) = x[s];
                }
            }
            ss += u[e].x * u[e].x + u[e].y * u[e].y + u[e].z * u[e].z + u[e].w * u[e].w;
        }
    }
    if (!a.h) return;
    float r = 1.f;
    if (a.weight) r = 1.0f / sqrtf(block_sum(ss, red) / (float)a.W + a.eps);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const int i = tid + e * nt;
        if (i >= nv) continue;
        float4 f = make_float4(u[e].x * r, u[e].y * r, u[e].z * r, u[e].w * r);
        if (a.weight) {
            const float4 w = bo_load4(a.weight, a.w_dtype == PE_F32, 4 * i);
            f.x *= w.x; f.y *= w.y; f.z *= w.z; f.w *= w.w;
        }
        if constexpr (sizeof(TH) == 4) *reinterpret_cast<float4*>((float*)a.h + t * a.W + 4 * i) = f;
        else {
            uint2 o;
            *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(f.x, f.y);
            *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(f.z, f.w);
            *reinterpret_cast<uint2*>((bf16*)a.h + t * a.W + 4 * i) = o;
        }
    }
}

#define SM_MAX_STREAMS 32
// Any width (one the shared memory holds a float32 row of) and up to 32 streams: a column a thread and step.
template <typename TH>
__global__ void __launch_bounds__(256) stream_mix_kernel(StreamArgs a) {
    pdl_launch_dependents();
    extern __shared__ float u[];
    __shared__ float red[33];
    pdl_wait();
    const size_t t = blockIdx.x;
    const int S = a.S, W = a.W;
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        float x[SM_MAX_STREAMS];
        for (int s = 0; s < S; ++s) x[s] = a.src[t * a.src_tok + s * a.src_stream + c];
        float sum = 0.f;
        if (a.y) {
            const float y = load_as_f(a.y, a.y_dtype, t * W + c);
            for (int to = 0; to < S; ++to) {
                float n = a.out[to] * y;
                for (int s = 0; s < S; ++s) n = fmaf(a.mix[s * S + to], x[s], n);
                if (a.dst) a.dst[(t * S + to) * W + c] = n;
                sum = a.in ? fmaf(a.in[to], n, sum) : sum + n;
            }
        } else {
            for (int s = 0; s < S; ++s) {
                sum = a.in ? fmaf(a.in[s], x[s], sum) : sum + x[s];
                if (a.dst) a.dst[(t * S + s) * W + c] = x[s];
            }
        }
        u[c] = sum;
        ss = fmaf(sum, sum, ss);
    }
    if (!a.h) return;
    const float r = a.weight ? 1.0f / sqrtf(block_sum(ss, red) / (float)W + a.eps) : 1.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x)                      // a thread reads back what it wrote itself
        ((TH*)a.h)[t * W + c] = from_f<TH>(u[c] * r * (a.weight ? load_as_f(a.weight, a.w_dtype, c) : 1.f));
}

extern "C" int pe_stream_mix(const float* src, long long src_tok, long long src_stream, float* dst, const void* y, int y_dtype, const float* mix,
                             const float* out, const float* in, const void* weight, int w_dtype, float eps, void* h, int h_dtype, int T, int S, int W,
                             void* stream) {
    if (T <= 0) return 0;
    if (S < 1 || S > SM_MAX_STREAMS || W < 1 || (y && (!mix || !out)) || (!dst && !h) || (h && h_dtype != PE_F32 && h_dtype != PE_BF16)) return PE_ERR_UNSUPPORTED;
    StreamArgs a = {src, src_tok, src_stream, dst, y, y_dtype, mix, out, in, weight, w_dtype, eps, h, S, W};
    cudaStream_t s = (cudaStream_t)stream;
    const bool x4 = S <= 8 && W % 4 == 0 && W <= 4096 && src_tok % 4 == 0 && src_stream % 4 == 0 &&
                    !(((uintptr_t)src | (uintptr_t)dst | (uintptr_t)y | (uintptr_t)weight | (uintptr_t)h) & 15);
    if (x4) {
        const int nv = W / 4, threads = nv >= 256 ? 256 : (nv + 31) / 32 * 32;
#define SM_GO(N) case N: if (h_dtype == PE_BF16 && h) PE_TRY(pe_launch(stream_mix_x4_kernel<N, bf16>, T, threads, 0, s, a)); \
                         else PE_TRY(pe_launch(stream_mix_x4_kernel<N, float>, T, threads, 0, s, a)); break;
        switch (S) { SM_GO(1) SM_GO(2) SM_GO(3) SM_GO(4) SM_GO(5) SM_GO(6) SM_GO(7) SM_GO(8) }
#undef SM_GO
    } else {
        const size_t smem = (size_t)W * 4;
        if (smem > 200 * 1024) return PE_ERR_UNSUPPORTED;
        if (h && h_dtype == PE_BF16) {
            PE_TRY(cudaFuncSetAttribute(stream_mix_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            PE_TRY(pe_launch(stream_mix_kernel<bf16>, T, 256, smem, s, a));
        } else {
            PE_TRY(cudaFuncSetAttribute(stream_mix_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
            PE_TRY(pe_launch(stream_mix_kernel<float>, T, 256, smem, s, a));
        }
    }
    PE_LAUNCH_CHECK();
    return 0;
}

// masked_attention.cu -- softmax or sigmoid attention with grouped key/value heads over the paged KV pools for a RAGGED batch
// (prompt portions and single decoded tokens in one launch), with the score modifiers and visibility rules a design
// picks by parameter:
//
//   score   s = (q . k) * scale;  softcap > 0: s <- softcap * tanh(s / softcap);  then a distance bias is added:
//           bias_kind 1: - slope[h] * (i - j)            (one slope per query head)
//           bias_kind 2: + table[min(i - j, len - 1)][h] (a table over the distance, one column per query head)
//           head_scale != null: s <- s * head_scale[h] right after the scale (a temperature per query head)
//           key_scale != null: the dot product is first multiplied by a number per cached key (the inverse root mean
//           square of a key that is cached before its norm)
//           head_bias != null: + head_bias[h], last
//   weight  softmax over the visible keys, or (sigm) sigmoid(s) of every visible key, with no sum to divide by
//   mask    mask_kind 0: causal (j <= i);  1: sliding window (0 <= i - j < size), which with mask_keep > 0 also keeps the
//           first mask_keep positions of the sequence visible (at their true positions);  2: chunks (j <= i and
//           floor(i / size) == floor(j / size), chunks counted from position 0 of the sequence)
//   sink    sink != null: exp(sink[h]) joins the softmax denominator of head h (a logit without key or value; zeros
//           give the "one added to the denominator" form)
//   output  out_rot != null: [rows][vdim / 2][cos, sin] of the batch rows; the neighbouring pairs (2m, 2m + 1) of every
//           head's output are turned BACK by the row's angle (values that were cached turned by their own position), in
//           float, before the result is rounded
//           gate != null: multiplied element by element by sigmoid(gate row), in float, before the result is rounded
//   values  v_pool == k_pool (and vdim == dim): the values ARE the cached key rows; the pool holds one row per key
//

// No rotation: positions enter through the bias and the mask only.  Scores, the modifiers, softmax weights and the
// weighted sums are float; K/V pages are stored in the activation type (float or bfloat16).  Only the key steps a
// tile's rows can see are visited, so the work per token is bounded by the window or chunk size.
//
// Pools: K pages [total_pages][tile_size][dim], V pages [total_pages][tile_size][vdim]; a (slot, kv head, tile) entry
// of the page table names the page of both (appended by pa_kv_append_rows).
#include "seq_common.cuh"

namespace pa {

// ---- rotation of this step's q | k | v rows fused with the append ----------------------------------------------------
// One warp per (row, unit): units [0, heads) are the query heads, rotated in place over their first rot_dims dimensions;
// units [heads, heads + kv_heads) are the key/value heads of a layer with a pool of its own: the key goes to its place in
// the pool rotated the same way, the value turned over all of vdim (vrot != null) or as it is.  Pairs are neighbours
// (2m, 2m + 1); the tables hold [rows][dims / 2][cos, sin] of the batch rows.
template <typename T>
__device__ __forceinline__ void ma_turn_copy(const T* __restrict__ src, T* __restrict__ dst, int n, int dims,
                                             const float* __restrict__ t, int lane) {
    for (int d = 2 * lane; d < n; d += 64) {
        float u = to_f32<T>(src[d]), v = d + 1 < n ? to_f32<T>(src[d + 1]) : 0.f;
        if (t && d + 1 < dims) {
            const float c = t[d], sn = t[d + 1];          // pair d / 2: entries (d / 2) * 2 and + 1
            const float u0 = u;
            u = u0 * c - v * sn;
            v = v * c + u0 * sn;
        }
        dst[d] = from_f32<T>(u);
        if (d + 1 < n) dst[d + 1] = from_f32<T>(v);
    }
}

template <typename T>
__global__ void rope_kv_append_kernel(T* __restrict__ src, int64_t stride, int q_off, int k_off, int v_off, int heads,
                                      int kv_heads, int dim, int vdim, int rot_dims, const float* __restrict__ rope,
                                      const float* __restrict__ vrot, T* __restrict__ k_pool, T* __restrict__ v_pool,
                                      const int32_t* __restrict__ table, int num_slots, int num_tiles, int total_pages,
                                      int tile_size, const int32_t* __restrict__ row_slot,
                                      const int32_t* __restrict__ row_pos, int rows) {
    const int lane = threadIdx.x & 31;
    const int units = heads + (k_pool ? kv_heads : 0);
    const int64_t w = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    if (w >= (int64_t)rows * units) return;
    const int u = (int)(w % units);
    const int64_t r = w / units;
    T* row = src + r * stride;
    const float* rt = rope ? rope + r * (rot_dims >> 1) * 2 : nullptr;
    if (u < heads) {
        if (rt) ma_turn_copy<T>(row + q_off + (int64_t)u * dim, row + q_off + (int64_t)u * dim, rot_dims, rot_dims, rt, lane);
        return;
    }
    const int g = u - heads;
    const int slot = row_slot[r], pos = row_pos[r];
    if (pos < 0 || pos / tile_size >= num_tiles || (unsigned)slot >= (unsigned)num_slots) return;
    const int page = table[((int64_t)slot * kv_heads + g) * num_tiles + pos / tile_size];
    if (page < 0 || page >= total_pages) return;
    const int64_t prow = (int64_t)page * tile_size + pos % tile_size;
    ma_turn_copy<T>(row + k_off + (int64_t)g * dim, k_pool + prow * dim, dim, rot_dims, rt, lane);
    ma_turn_copy<T>(row + v_off + (int64_t)g * vdim, v_pool + prow * vdim, vdim, vdim,
                    vrot ? vrot + r * (vdim >> 1) * 2 : nullptr, lane);
}

// ---- query / key norm of this step's rows fused with the append --------------------------------------------------------
// One warp per (row, unit): units [0, heads) are the query heads, divided by their root mean square and multiplied by
// q_gain, in place; units [heads, heads + kv_heads) are the key/value heads.  key_scale == null: the key goes to its place
// in the pool normed (k_gain).  key_scale != null: the key goes there as projected and its inverse root mean square to
// key_scale, so the pool row can serve as the value too (the key norm's gain is then part of q_gain: only the product of
// the two enters a score).  v_pool != null: a value row of its own, as it is.
template <typename T>
__device__ __forceinline__ float qk_inv_rms(const T* __restrict__ x, int dim, float eps, int lane) {
    float ss = 0.f;
    for (int d = lane; d < dim; d += 32) {
        const float v = to_f32<T>(x[d]);
        ss = fmaf(v, v, ss);
    }
    return 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
}

template <typename T>
__global__ void __launch_bounds__(256) qk_norm_kv_append_kernel(T* __restrict__ src, int64_t stride, int q_off, int k_off, int v_off,
                                         int heads, int kv_heads, int dim, int vdim, const float* __restrict__ q_gain,
                                         const float* __restrict__ k_gain, float eps, T* __restrict__ k_pool,
                                         T* __restrict__ v_pool, float* __restrict__ key_scale,
                                         const int32_t* __restrict__ table, int num_slots, int num_tiles, int total_pages,
                                         int tile_size, const int32_t* __restrict__ row_slot,
                                         const int32_t* __restrict__ row_pos, int rows) {
    const int lane = threadIdx.x & 31;
    const int units = heads + kv_heads;
    const int64_t w = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    if (w >= (int64_t)rows * units) return;
    const int u = (int)(w % units);
    const int64_t r = w / units;
    T* row = src + r * stride;
    if (u < heads) {
        T* q = row + q_off + (int64_t)u * dim;
        const float rn = qk_inv_rms<T>(q, dim, eps, lane);
        for (int d = lane; d < dim; d += 32) q[d] = from_f32<T>(to_f32<T>(q[d]) * rn * q_gain[d]);
        return;
    }
    const int g = u - heads;
    const int slot = row_slot[r], pos = row_pos[r];
    if (pos < 0 || pos / tile_size >= num_tiles || (unsigned)slot >= (unsigned)num_slots) return;
    const int page = table[((int64_t)slot * kv_heads + g) * num_tiles + pos / tile_size];
    if (page < 0 || page >= total_pages) return;
    const int64_t prow = (int64_t)page * tile_size + pos % tile_size;
    const T* k = row + k_off + (int64_t)g * dim;
    const float rn = qk_inv_rms<T>(k, dim, eps, lane);
    T* kd = k_pool + prow * dim;
    if (key_scale) {
        for (int d = lane; d < dim; d += 32) kd[d] = k[d];
        if (lane == 0) key_scale[prow] = rn;
    } else {
        for (int d = lane; d < dim; d += 32) kd[d] = from_f32<T>(to_f32<T>(k[d]) * rn * k_gain[d]);
    }
    if (v_pool) {
        const T* v = row + v_off + (int64_t)g * vdim;
        for (int d = lane; d < vdim; d += 32) v_pool[prow * vdim + d] = v[d];
    }
}

// ---- short convolution, rotation and norm of this step's q | k | v rows fused with the append -----------------------------
// One warp per (work item, unit): an item is a run of consecutive tokens of one portion, units are the query heads, the key
// heads and the value heads (the latter two only where the layer has a pool of its own).  Per token and channel
//     y_t = sum_b w[b] u_(t - b)      (b tokens back; w == null: y_t = u_t)
// over the RAW projected rows u (before the portion: the state slot's last taps - 1 rows), accumulated in float; queries and
// keys are then rotated over their first rot_dims dimensions (neighbouring pairs) and, with `norm`, divided by their root
// mean square over dim -- both still in float, one rounding at the end.  Queries go to q_out, keys and values to their place
// in the pools.  A lane owns the pairs (2 lane + 64 i, + 1) and slides a window of inputs along the item, so every raw row
// is read once per item (plus the taps - 1 rows before it).  The items that START a portion leave the state for the next
// step: they are the only readers of the slot's old rows, channel by channel in the same thread.
struct ConvAppendParams {
    const void* in;             // raw rows [q | k | v] from column in_off
    int64_t in_stride;
    int in_off, channels, heads, kv_heads, dim, vdim, rot_dims, taps;
    const float* w;             // [taps][channels], entry b = the weight b tokens back, or null
    float* state;               // [slots][taps - 1][channels], oldest row first
    const float* rope;          // [rows][rot_dims / 2][cos, sin] of the batch rows
    int norm;
    float eps;
    void* q_out;
    int64_t q_out_stride;
    void* k_pool;
    void* v_pool;
    const int32_t* table;
    int num_slots, num_tiles, total_pages, tile_size;
    const int32_t* items;       // [n][6]: first row, tokens, slot, offset within the portion, portion's length, first position
    int num_items;
    int pairs;                  // every pair of columns starts on a boundary of two elements
    int words;                  // 4 or 8: heads are whole words of that many columns, everything aligned: the vector form
};
constexpr int kCaMaxTaps = 8;

template <typename T>
__device__ __forceinline__ void ca_load(const T* __restrict__ p, int pairs, bool second, float& u, float& v) {
    if (pairs) {
        if constexpr (sizeof(T) == 2) {
            const uint32_t w = *reinterpret_cast<const uint32_t*>(p);
            u = __uint_as_float(w << 16);
            v = __uint_as_float(w & 0xffff0000u);
        } else {
            const float2 w = *reinterpret_cast<const float2*>(p);
            u = w.x;
            v = w.y;
        }
    } else {
        u = to_f32<T>(p[0]);
        v = second ? to_f32<T>(p[1]) : 0.f;
    }
}
template <typename T>
__device__ __forceinline__ void ca_store(T* __restrict__ p, int pairs, bool second, float u, float v) {
    if (pairs) {
        if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(u, v);
        else *reinterpret_cast<float2*>(p) = make_float2(u, v);
    } else {
        p[0] = from_f32<T>(u);
        if (second) p[1] = from_f32<T>(v);
    }
}

// NP: pairs per lane; TAPS: padded taps (the weights past `taps` are zero)
template <typename T, int NP, int TAPS>
__global__ void __launch_bounds__(256) conv_rope_norm_append_kernel(const ConvAppendParams p) {
    const int lane = threadIdx.x & 31;
    const int units = p.heads + (p.k_pool ? 2 * p.kv_heads : 0);
    const int64_t wid = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
    if (wid >= (int64_t)p.num_items * units) return;
    const int unit = (int)(wid % units);
    const int* it = p.items + 6 * (wid / units);
    const int row0 = it[0], n = it[1], slot = it[2], off = it[3], plen = it[4], pos0 = it[5];
    if ((unsigned)slot >= (unsigned)p.num_slots) return;
    const int kind = unit < p.heads ? 0 : unit < p.heads + p.kv_heads ? 1 : 2;       // query, key, value
    const int g = kind == 0 ? 0 : unit - p.heads - (kind - 1) * p.kv_heads;
    const int size = kind == 2 ? p.vdim : p.dim;
    const int ch0 = kind == 0 ? unit * p.dim : p.heads * p.dim + (kind == 1 ? g * p.dim : p.kv_heads * p.dim + g * p.vdim);
    const T* in = static_cast<const T*>(p.in) + p.in_off + ch0;
    const int taps = p.w ? p.taps : 1;
    float* st = taps > 1 ? p.state + (int64_t)slot * (taps - 1) * p.channels + ch0 : nullptr;
    const int32_t* trow = kind ? p.table + ((int64_t)slot * p.kv_heads + g) * p.num_tiles : nullptr;

    float wt[TAPS][NP][2], win[TAPS][NP][2], nxt[NP][2];
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int d = 2 * lane + 64 * i;
#pragma unroll
        for (int b = 0; b < TAPS; ++b) {
            wt[b][i][0] = wt[b][i][1] = 0.f;
            win[b][i][0] = win[b][i][1] = 0.f;
        }
        nxt[i][0] = nxt[i][1] = 0.f;
        if (d >= size) continue;
        const bool second = d + 1 < size;
        if (p.w) {
#pragma unroll
            for (int b = 0; b < TAPS; ++b)
                if (b < taps) {
                    wt[b][i][0] = p.w[(int64_t)b * p.channels + ch0 + d];
                    if (second) wt[b][i][1] = p.w[(int64_t)b * p.channels + ch0 + d + 1];
                }
        } else {
            wt[0][i][0] = wt[0][i][1] = 1.f;
        }
        // win[b] = the input b tokens before the CURRENT one; entering the loop it is shifted once
#pragma unroll
        for (int b = 0; b + 1 < TAPS; ++b)
            if (b < taps - 1) {
                const int t = off - 1 - b;             // offset within the portion
                if (t >= 0) {
                    ca_load<T>(in + (int64_t)(row0 - 1 - b) * p.in_stride + d, p.pairs, second, win[b][i][0], win[b][i][1]);
                } else {
                    win[b][i][0] = st[(int64_t)(taps - 1 + t) * p.channels + d];
                    if (second) win[b][i][1] = st[(int64_t)(taps - 1 + t) * p.channels + d + 1];
                }
            }
        ca_load<T>(in + (int64_t)row0 * p.in_stride + d, p.pairs, second, nxt[i][0], nxt[i][1]);
    }

    for (int t = 0; t < n; ++t) {
        const int64_t r = row0 + t;
        float y[NP][2];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int d = 2 * lane + 64 * i;
#pragma unroll
            for (int b = TAPS - 1; b > 0; --b) {
                win[b][i][0] = win[b - 1][i][0];
                win[b][i][1] = win[b - 1][i][1];
            }
            win[0][i][0] = nxt[i][0];
            win[0][i][1] = nxt[i][1];
            if (t + 1 < n && d < size)                 // the next token's row is on its way while this one is computed
                ca_load<T>(in + (r + 1) * p.in_stride + d, p.pairs, d + 1 < size, nxt[i][0], nxt[i][1]);
            float u = 0.f, v = 0.f;
#pragma unroll
            for (int b = 0; b < TAPS; ++b) {
                u = fmaf(wt[b][i][0], win[b][i][0], u);
                v = fmaf(wt[b][i][1], win[b][i][1], v);
            }
            if (kind < 2 && d < p.rot_dims) {
                const float2 cs = *reinterpret_cast<const float2*>(p.rope + r * p.rot_dims + d);
                const float u0 = u;
                u = u0 * cs.x - v * cs.y;
                v = v * cs.x + u0 * cs.y;
            }
            y[i][0] = u;
            y[i][1] = v;
            ss = fmaf(u, u, fmaf(v, v, ss));
        }
        if (kind < 2 && p.norm) {
            const float rn = 1.0f / sqrtf(warp_sum(ss) / (float)size + p.eps);
#pragma unroll
            for (int i = 0; i < NP; ++i) { y[i][0] *= rn; y[i][1] *= rn; }
        }
        T* dst;
        if (kind == 0) {
            dst = static_cast<T*>(p.q_out) + r * p.q_out_stride + ch0;
        } else {
            const int pos = pos0 + t;
            if (pos < 0 || pos / p.tile_size >= p.num_tiles) continue;
            const int page = trow[pos / p.tile_size];
            if (page < 0 || page >= p.total_pages) continue;
            const int64_t prow = (int64_t)page * p.tile_size + pos % p.tile_size;
            dst = static_cast<T*>(kind == 1 ? p.k_pool : p.v_pool) + prow * size;
        }
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int d = 2 * lane + 64 * i;
            if (d < size) ca_store<T>(dst + d, p.pairs, d + 1 < size, y[i][0], y[i][1]);
        }
    }

    if (off != 0 || taps <= 1) return;
    // the portion's last taps - 1 raw rows become the state; rows older than the portion move up within the slot
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int d = 2 * lane + 64 * i;
        if (d >= size) continue;
        const bool second = d + 1 < size;
        for (int j = 0; j < taps - 1; ++j) {
            const int t = plen - (taps - 1) + j;
            float u, v = 0.f;
            if (t >= 0) {
                ca_load<T>(in + (int64_t)(row0 + t) * p.in_stride + d, p.pairs, second, u, v);
            } else {
                u = st[(int64_t)(taps - 1 + t) * p.channels + d];
                if (second) v = st[(int64_t)(taps - 1 + t) * p.channels + d + 1];
            }
            st[(int64_t)j * p.channels + d] = u;
            if (second) st[(int64_t)j * p.channels + d + 1] = v;
        }
    }
}

// The same for heads of at most 256 whose rows are whole words of EPL columns: a unit is LANES lanes with EPL neighbouring
// columns each (the pairs of a rotation lie within a lane), 32 / LANES units per warp.  The raw rows of the next kAhead tokens
// and the rotation of the next one are on their way while the current one is computed; the page of a row is looked up when a
// new page begins.  The window is a ring of TAPS rows: the loop is unrolled over kAhead tokens (a multiple of TAPS), so
// every place in it is fixed at compile time.
constexpr int kCaThreads = 128;

template <typename T, int EPL> struct CaWord { uint32_t w[EPL * sizeof(T) / 4]; };
template <typename T, int EPL>
__device__ __forceinline__ CaWord<T, EPL> ca_word_load(const T* __restrict__ p) {
    CaWord<T, EPL> r;
    if constexpr (EPL * sizeof(T) == 8) {
        const uint2 v = *reinterpret_cast<const uint2*>(p);
        r.w[0] = v.x; r.w[1] = v.y;
    } else {
#pragma unroll
        for (int i = 0; i < (int)(EPL * sizeof(T) / 16); ++i) {
            const uint4 v = reinterpret_cast<const uint4*>(p)[i];
            r.w[4 * i] = v.x; r.w[4 * i + 1] = v.y; r.w[4 * i + 2] = v.z; r.w[4 * i + 3] = v.w;
        }
    }
    return r;
}
template <typename T, int EPL>
__device__ __forceinline__ void ca_word_unpack(const CaWord<T, EPL>& r, float (&f)[EPL]) {
    if constexpr (sizeof(T) == 2) {
#pragma unroll
        for (int i = 0; i < EPL / 2; ++i) {
            f[2 * i] = __uint_as_float(r.w[i] << 16);
            f[2 * i + 1] = __uint_as_float(r.w[i] & 0xffff0000u);
        }
    } else {
#pragma unroll
        for (int i = 0; i < EPL; ++i) f[i] = __uint_as_float(r.w[i]);
    }
}
template <typename T, int EPL>
__device__ __forceinline__ void ca_word_store(T* __restrict__ p, const float (&f)[EPL]) {
    if constexpr (sizeof(T) == 2 && EPL == 4) {
        *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
    } else if constexpr (sizeof(T) == 2) {
        *reinterpret_cast<uint4*>(p) = bf16x8_pack(f);
    } else {
#pragma unroll
        for (int i = 0; i < EPL / 4; ++i) reinterpret_cast<float4*>(p)[i] = make_float4(f[4 * i], f[4 * i + 1], f[4 * i + 2], f[4 * i + 3]);
    }
}
template <int EPL>
__device__ __forceinline__ void ca_load_floats(const float* __restrict__ p, float (&f)[EPL]) {
#pragma unroll
    for (int i = 0; i < EPL / 4; ++i) {
        const float4 a = reinterpret_cast<const float4*>(p)[i];
        f[4 * i] = a.x; f[4 * i + 1] = a.y; f[4 * i + 2] = a.z; f[4 * i + 3] = a.w;
    }
}

template <typename T, int EPL, int LANES, int TAPS>
__global__ void __launch_bounds__(kCaThreads, EPL == 4 && TAPS <= 4 ? 5 : 1) conv_rope_norm_append_vec_kernel(const ConvAppendParams p) {
    constexpr int kAhead = TAPS < 4 ? 4 : TAPS;
    const int lane = threadIdx.x & (LANES - 1);
    const int units = p.heads + (p.k_pool ? 2 * p.kv_heads : 0);
    const uint32_t uid = (blockIdx.x * (uint32_t)blockDim.x + threadIdx.x) / LANES;
    // every lane of a warp stays to the end (the sums over a unit's lanes are warp shuffles); lanes past the last unit or past
    // a head's size read its first columns and write nothing
    const bool unit_ok = uid < (uint32_t)p.num_items * (uint32_t)units;
    const int item = unit_ok ? (int)(uid / units) : 0, unit = unit_ok ? (int)(uid % units) : 0;
    const int* it = p.items + 6 * item;
    const int row0 = it[0], n = it[1], off = it[3], plen = it[4], pos0 = it[5];
    const int kind = unit < p.heads ? 0 : unit < p.heads + p.kv_heads ? 1 : 2;       // query, key, value
    const int g = kind == 0 ? 0 : unit - p.heads - (kind - 1) * p.kv_heads;
    const int size = kind == 2 ? p.vdim : p.dim;
    const bool slot_ok = (unsigned)it[2] < (unsigned)p.num_slots;
    const bool live = unit_ok && lane * EPL < size && slot_ok;
    const int slot = slot_ok ? it[2] : 0;
    const int d = lane * EPL < size ? lane * EPL : 0;
    const int ch0 = (kind == 0 ? unit * p.dim : p.heads * p.dim + (kind == 1 ? g * p.dim : p.kv_heads * p.dim + g * p.vdim)) + d;
    const int stride = (int)p.in_stride;
    const T* in = static_cast<const T*>(p.in) + p.in_off + ch0 + (int64_t)row0 * stride;
    const int taps = p.w ? p.taps : 1;
    float* st = taps > 1 ? p.state + (int64_t)slot * (taps - 1) * p.channels + ch0 : nullptr;
    const int turned = kind < 2 ? min(EPL, max(0, p.rot_dims - d)) : 0;      // columns of this lane that are rotated
    const float* rp = p.rope + (int64_t)row0 * p.rot_dims + d;
    const bool norm = kind < 2 && p.norm;
    const float inv_size = 1.0f / (float)size;

    CaWord<T, EPL> nxt[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i) nxt[i] = ca_word_load<T, EPL>(in + (int64_t)min(i, n - 1) * stride);
    float cs[EPL];                                     // cos, sin of this lane's pairs at the current token
#pragma unroll
    for (int c = 0; c < EPL; ++c) cs[c] = 0.f;
    auto load_turn = [&]() {
#pragma unroll
        for (int c = 0; c < EPL; c += 4)
            if (c < turned) {
                const float4 v = *reinterpret_cast<const float4*>(rp + c);
                cs[c] = v.x; cs[c + 1] = v.y; cs[c + 2] = v.z; cs[c + 3] = v.w;
            }
        rp += p.rot_dims;
    };
    load_turn();
    float wt[TAPS][EPL], win[TAPS][EPL];               // win: ring, token t in place t % TAPS
#pragma unroll
    for (int b = 0; b < TAPS; ++b)
#pragma unroll
        for (int c = 0; c < EPL; ++c) {
            wt[b][c] = p.w ? 0.f : b == 0 ? 1.f : 0.f;
            win[b][c] = 0.f;
        }
    if (p.w) {
#pragma unroll
        for (int b = 0; b < TAPS; ++b)
            if (b < taps) ca_load_floats<EPL>(p.w + (int64_t)b * p.channels + ch0, wt[b]);
    }
#pragma unroll
    for (int b = 1; b < TAPS; ++b)
        if (b < taps) {
            const int t = off - b;                     // offset within the portion
            if (t >= 0) ca_word_unpack<T, EPL>(ca_word_load<T, EPL>(in - (int64_t)b * stride), win[TAPS - b]);
            else ca_load_floats<EPL>(st + (int64_t)(taps - 1 + t) * p.channels, win[TAPS - b]);
        }
    // destination of the current token's row (null: not stored), and its place in its page
    T* dst = kind == 0 ? static_cast<T*>(p.q_out) + (int64_t)row0 * p.q_out_stride + ch0 : nullptr;
    const int64_t dstep = kind == 0 ? p.q_out_stride : size;
    int tile = 0, at = 0;
    auto look_up = [&]() {
        const int page = tile < p.num_tiles ? p.table[((int64_t)slot * p.kv_heads + g) * p.num_tiles + tile] : -1;
        dst = page >= 0 && page < p.total_pages
                  ? static_cast<T*>(kind == 1 ? p.k_pool : p.v_pool) + ((int64_t)page * p.tile_size + at) * size + d : nullptr;
    };
    if (kind && pos0 >= 0) {
        tile = pos0 / p.tile_size;
        at = pos0 - tile * p.tile_size;
        look_up();
    }

    for (int t0 = 0; t0 < n; t0 += kAhead) {         // units of a warp with fewer tokens leave the loop as a whole
#pragma unroll
        for (int i = 0; i < kAhead; ++i) {
            const int t = t0 + i;
            if (t >= n) break;
            float y[EPL];
            float (&now)[EPL] = win[i % TAPS];
            ca_word_unpack<T, EPL>(nxt[i], now);
            if (t + kAhead < n) nxt[i] = ca_word_load<T, EPL>(in + (int64_t)(t + kAhead) * stride);
#pragma unroll
            for (int c = 0; c < EPL; ++c) {
                y[c] = wt[0][c] * now[c];
#pragma unroll
                for (int b = 1; b < TAPS; ++b) y[c] = fmaf(wt[b][c], win[(i + TAPS - b) % TAPS][c], y[c]);
            }
#pragma unroll
            for (int c = 0; c < EPL; c += 4)
                if (c < turned) {
                    const float u0 = y[c], v0 = y[c + 1], u1 = y[c + 2], v1 = y[c + 3];
                    y[c] = u0 * cs[c] - v0 * cs[c + 1];
                    y[c + 1] = v0 * cs[c] + u0 * cs[c + 1];
                    y[c + 2] = u1 * cs[c + 2] - v1 * cs[c + 3];
                    y[c + 3] = v1 * cs[c + 2] + u1 * cs[c + 3];
                }
            if (t + 1 < n) load_turn();
            if (norm) {
                float ss = 0.f;
#pragma unroll
                for (int c = 0; c < EPL; ++c) ss = fmaf(y[c], y[c], ss);
                if (lane * EPL >= size) ss = 0.f;
                const unsigned mask = LANES == 32 ? 0xffffffffu : ((1u << LANES) - 1u) << (threadIdx.x & 31 & ~(LANES - 1));
#pragma unroll
                for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
                const float rn = rsqrtf(fmaf(ss, inv_size, p.eps));
#pragma unroll
                for (int c = 0; c < EPL; ++c) y[c] *= rn;
            }
            if (live && dst) ca_word_store<T, EPL>(dst, y);
            if (dst) dst += dstep;
            if (kind && ++at == p.tile_size) {
                at = 0;
                ++tile;
                if (t + 1 < n) look_up();
            }
        }
    }

    if (!live || off != 0 || taps <= 1) return;
    for (int j = 0; j < taps - 1; ++j) {               // rows older than the portion move up within the slot
        const int t = plen - (taps - 1) + j;
        float f[EPL];
        if (t >= 0) ca_word_unpack<T, EPL>(ca_word_load<T, EPL>(in + (int64_t)t * stride), f);
        else ca_load_floats<EPL>(st + (int64_t)(taps - 1 + t) * p.channels, f);
        ca_word_store<float, EPL>(st + (int64_t)j * p.channels, f);
    }
}

template <typename T, int EPL, int LANES>
static int ca_launch_vec(const ConvAppendParams& p, cudaStream_t st) {
    const int units = p.heads + (p.k_pool ? 2 * p.kv_heads : 0);
    const unsigned grid = (unsigned)(((int64_t)p.num_items * units * LANES + kCaThreads - 1) / kCaThreads);
    const int taps = p.w ? p.taps : 1;
    if (taps <= 1) conv_rope_norm_append_vec_kernel<T, EPL, LANES, 1><<<grid, kCaThreads, 0, st>>>(p);
    else if (taps <= 4) conv_rope_norm_append_vec_kernel<T, EPL, LANES, 4><<<grid, kCaThreads, 0, st>>>(p);
    else conv_rope_norm_append_vec_kernel<T, EPL, LANES, kCaMaxTaps><<<grid, kCaThreads, 0, st>>>(p);
    PA_RETURN_LAUNCH_STATUS();
}

template <typename T, int NP>
static int ca_launch(const ConvAppendParams& p, cudaStream_t st) {
    const int units = p.heads + (p.k_pool ? 2 * p.kv_heads : 0);
    const unsigned grid = (unsigned)(((int64_t)p.num_items * units * 32 + 255) / 256);
    const int taps = p.w ? p.taps : 1;
    if (taps <= 1) conv_rope_norm_append_kernel<T, NP, 1><<<grid, 256, 0, st>>>(p);
    else if (taps <= 4) conv_rope_norm_append_kernel<T, NP, 4><<<grid, 256, 0, st>>>(p);
    else conv_rope_norm_append_kernel<T, NP, kCaMaxTaps><<<grid, 256, 0, st>>>(p);
    PA_RETURN_LAUNCH_STATUS();
}

template <typename T>
static int ca_dispatch(const ConvAppendParams& p, cudaStream_t st) {
    const int n = p.k_pool && p.vdim > p.dim ? p.vdim : p.dim;
    if (p.words >= 4 && n <= 128) {
        if (n <= 32) return ca_launch_vec<T, 4, 8>(p, st);
        if (n <= 64) return ca_launch_vec<T, 4, 16>(p, st);
        return ca_launch_vec<T, 4, 32>(p, st);
    }
    if (p.words == 8 && n <= 256) return ca_launch_vec<T, 8, 32>(p, st);
    if (n <= 64) return ca_launch<T, 1>(p, st);
    if (n <= 128) return ca_launch<T, 2>(p, st);
    if (n <= 256) return ca_launch<T, 4>(p, st);
    if (n <= 512) return ca_launch<T, 8>(p, st);
    return PA_ERR_UNSUPPORTED;
}

constexpr int kMaRows = 32;     // (token, head) rows per CTA
constexpr int kMaWarps = 8;
constexpr int kMaRpw = kMaRows / kMaWarps;
constexpr int kMaKeys = 32;     // keys staged per step

struct MaskAttnParams {
    const void* q;              // rows of the projection buffer; the query of head h starts at q_off + h * dim
    int64_t q_stride;
    int q_off;
    const void* k_pool;
    const void* v_pool;
    const int32_t* table;
    int num_slots, num_kv_heads, num_tiles, total_pages, tile_size;
    const int32_t* tiles;       // [ntiles][4]: first row, tokens, slot, position of the first token
    int heads, dim, vdim;
    float scale, softcap;
    int mask_kind, mask_size;
    int bias_kind, bias_len;
    const float* bias;          // kind 1: [heads]; kind 2: [bias_len][heads]
    void* out;                  // [rows][heads * vdim]
    const float* head_scale;    // [heads] or null
    const float* sink;          // [heads] or null
    int mask_keep;              // window masks: the first mask_keep positions stay visible
    const float* out_rot;       // [rows][vdim / 2][2] or null
    int sigm;                   // 1: weight = sigmoid(score), nothing divides the sum (no sink)
    const float* key_scale;     // [total_pages * tile_size] or null
    const float* head_bias;     // [heads] or null
    const void* gate;           // rows of the activation type; the gate of output column c of head h at gate_off + h * vdim + c
    int64_t gate_stride;
    int gate_off;
};

__device__ __forceinline__ int ma_first_key(const MaskAttnParams& p, int pos) {
    if (p.mask_kind == 1) return max(0, pos - p.mask_size + 1);
    if (p.mask_kind == 2) return pos / p.mask_size * p.mask_size;
    return 0;
}

__device__ __forceinline__ bool ma_visible(const MaskAttnParams& p, int i, int j) {
    if (j > i) return false;
    if (p.mask_kind == 1) return i - j < p.mask_size || j < p.mask_keep;
    if (p.mask_kind == 2) return i / p.mask_size == j / p.mask_size;
    return true;
}

// The key steps (runs of `keys` positions) the rows of a tile can see, in order: the steps of the kept first positions,
// then the steps from the first key of the tile's first token (ma_first_key) to its last token.  `first` = that first
// key, `total` = keys up to the tile's last token.
struct MaSteps {
    int head, body0, count;
    __device__ __forceinline__ int step(int n) const { return n < head ? n : body0 + n - head; }
};
__device__ __forceinline__ MaSteps ma_steps(const MaskAttnParams& p, int first, int total, int keys) {
    MaSteps s;
    s.body0 = first / keys;
    s.head = 0;
    if (p.mask_kind == 1 && p.mask_keep > 0) s.head = min(s.body0, (min(p.mask_keep, total) + keys - 1) / keys);
    s.count = s.head + (total + keys - 1) / keys - s.body0;
    return s;
}

// the softmax denominator with the sink of head h: returns the factor for the accumulated sums (and updates l)
__device__ __forceinline__ float ma_sink(const MaskAttnParams& p, int h, float m, float& l) {
    if (!p.sink) return 1.f;
    const float sk = p.sink[h];
    const float n = fmaxf(m, sk);
    const float c = m == -INFINITY ? 0.f : expf(m - n);
    l = l * c + expf(sk - n);
    return c;
}

// turns the pair (u, v) = columns (2m, 2m + 1) of batch row `row` back by the row's angle; even = this thread holds u
__device__ __forceinline__ float ma_unturn(const MaskAttnParams& p, int64_t row, int col, float mine, float other) {
    const float* t = p.out_rot + (row * (p.vdim >> 1) + (col >> 1)) * 2;
    return (col & 1) ? mine * t[0] - other * t[1] : mine * t[0] + other * t[1];
}

// the float score of (query position i, key position j, query head h) from the raw dot product
__device__ __forceinline__ float ma_score(const MaskAttnParams& p, float dot, int i, int j, int h, float slope) {
    float s = dot * p.scale;
    if (p.head_scale) s *= p.head_scale[h];
    if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
    if (p.bias_kind == 1) s -= slope * (float)(i - j);
    else if (p.bias_kind == 2) s += p.bias[(int64_t)min(i - j, p.bias_len - 1) * p.heads + h];
    if (p.head_bias) s += p.head_bias[h];
    return s;
}

// the factor of output column `col` (of all heads' columns) of batch row `row`
template <typename T>
__device__ __forceinline__ float ma_gate(const MaskAttnParams& p, int64_t row, int col) {
    return sigmoid_f32(to_f32<T>(static_cast<const T*>(p.gate)[row * p.gate_stride + p.gate_off + col]));
}

__device__ __forceinline__ void ma_geometry(int heads, int kv_heads, int& hpg, int& hc, int& nchunk) {
    hpg = heads / kv_heads;
    hc = hpg < kMaRows ? hpg : kMaRows;
    nchunk = (hpg + hc - 1) / hc;
}

// CTA of 8 warps = 32 (token, head) rows that read the SAME key/value head: up to 32 / hc consecutive tokens of one
// portion x hc = min(32, heads per kv head) query heads.  Keys are staged 32 at a time (one key per lane for the
// scores; lanes switch to value columns for the weighted sums).
template <typename T, int NV>
__global__ void __launch_bounds__(kMaWarps * 32) masked_attention_kernel(const MaskAttnParams p) {
    extern __shared__ float smem[];
    const int kd = p.dim, kds = kd + 1;
    float* Qs = smem;                              // [32][kd]
    float* Ks = Qs + kMaRows * kd;                 // [32][kd + 1]
    float* Vs = Ks + kMaKeys * kds;                // [32][vdim]
    __shared__ int64_t page_row[kMaKeys];          // pool row of the staged key, or -1

    int hpg, hc, nchunk;
    ma_geometry(p.heads, p.num_kv_heads, hpg, hc, nchunk);
    const int bq = kMaRows / hc;
    const int* tile = p.tiles + 4 * blockIdx.x;
    const int row0 = tile[0], ntok = tile[1], slot = tile[2], pos0 = tile[3];
    const int g = blockIdx.y / nchunk, chunk = blockIdx.y % nchunk;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const T* kp = static_cast<const T*>(p.k_pool);
    const T* vp = static_cast<const T*>(p.v_pool);

    for (int idx = threadIdx.x; idx < kMaRows * kd; idx += blockDim.x) {
        const int r = idx / kd, d = idx % kd;
        const int tok = r / hc, hh = chunk * hc + r % hc;
        float v = 0.f;
        if (tok < bq && tok < ntok && hh < hpg)
            v = to_f32<T>(static_cast<const T*>(p.q)[(int64_t)(row0 + tok) * p.q_stride + p.q_off + (int64_t)(g * hpg + hh) * kd + d]);
        Qs[idx] = v;
    }

    int rpos[kMaRpw], rhead[kMaRpw];   // position of the row's token (-1: unused row) and its query head
    float slope[kMaRpw], m[kMaRpw], l[kMaRpw], acc[kMaRpw][NV];
#pragma unroll
    for (int r = 0; r < kMaRpw; ++r) {
        const int row = warp * kMaRpw + r;
        const int tok = row / hc, hh = chunk * hc + row % hc;
        const bool used = tok < bq && tok < ntok && hh < hpg;
        rpos[r] = used ? pos0 + tok : -1;
        rhead[r] = used ? g * hpg + hh : 0;
        slope[r] = p.bias_kind == 1 ? p.bias[rhead[r]] : 0.f;
        m[r] = -INFINITY;
        l[r] = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) acc[r][i] = 0.f;
    }

    const int last_tok = min(ntok, bq) - 1;
    const int total = pos0 + last_tok + 1;                 // keys any row of the tile may see
    const MaSteps steps = ma_steps(p, ma_first_key(p, pos0), total, kMaKeys);

    for (int sn = 0; sn < steps.count; ++sn) {
        const int c0 = steps.step(sn) * kMaKeys;
        __syncthreads();                                   // the previous step's tiles are consumed (and Qs is written)
        if (threadIdx.x < kMaKeys) {
            const int j = c0 + threadIdx.x;
            int64_t pr = -1;
            if (j < total && j / p.tile_size < p.num_tiles) {
                const int page = p.table[((int64_t)slot * p.num_kv_heads + g) * p.num_tiles + j / p.tile_size];
                if (page >= 0 && page < p.total_pages) pr = (int64_t)page * p.tile_size + j % p.tile_size;
            }
            page_row[threadIdx.x] = pr;
        }
        __syncthreads();
        for (int idx = threadIdx.x; idx < kMaKeys * kd; idx += blockDim.x) {
            const int key = idx / kd, d = idx % kd;
            const int64_t pr = page_row[key];
            Ks[key * kds + d] = pr >= 0 ? to_f32<T>(kp[pr * kd + d]) : 0.f;
        }
        for (int idx = threadIdx.x; idx < kMaKeys * p.vdim; idx += blockDim.x) {
            const int key = idx / p.vdim, d = idx % p.vdim;
            const int64_t pr = page_row[key];
            Vs[idx] = pr >= 0 ? to_f32<T>(vp[pr * p.vdim + d]) : 0.f;
        }
        __syncthreads();

        // ---- scores: lane = key
        float s[kMaRpw];
#pragma unroll
        for (int r = 0; r < kMaRpw; ++r) s[r] = 0.f;
        const float* kr = Ks + lane * kds;
        const float* qb = Qs + warp * kMaRpw * kd;
        for (int d = 0; d < kd; ++d) {
            const float kv = kr[d];
#pragma unroll
            for (int r = 0; r < kMaRpw; ++r) s[r] = fmaf(qb[r * kd + d], kv, s[r]);
        }
        const int j = c0 + lane;
        const bool mapped = page_row[lane] >= 0;
        const float ks = mapped && p.key_scale ? p.key_scale[page_row[lane]] : 1.f;
        float w[kMaRpw];
#pragma unroll
        for (int r = 0; r < kMaRpw; ++r) {
            const bool vis = mapped && rpos[r] >= 0 && ma_visible(p, rpos[r], j);
            const float v = vis ? ma_score(p, s[r] * ks, rpos[r], j, rhead[r], slope[r]) : -INFINITY;
            if (p.sigm) {
                w[r] = vis ? sigmoid_f32(v) : 0.f;
                continue;
            }
            const float n = fmaxf(m[r], warp_max(v));
            const float c = n == -INFINITY ? 1.f : expf(m[r] - n);
            w[r] = vis ? expf(v - n) : 0.f;
            l[r] = l[r] * c + warp_sum(w[r]);
            m[r] = n;
#pragma unroll
            for (int i = 0; i < NV; ++i) acc[r][i] *= c;
        }
        // ---- weighted sums: lane = value column
        const int nk = min(kMaKeys, total - c0);
        for (int jj = 0; jj < nk; ++jj) {
            float v[NV];
#pragma unroll
            for (int i = 0; i < NV; ++i) v[i] = lane + 32 * i < p.vdim ? Vs[jj * p.vdim + lane + 32 * i] : 0.f;
#pragma unroll
            for (int r = 0; r < kMaRpw; ++r) {
                const float wj = __shfl_sync(0xffffffffu, w[r], jj);
#pragma unroll
                for (int i = 0; i < NV; ++i) acc[r][i] = fmaf(wj, v[i], acc[r][i]);
            }
        }
    }

#pragma unroll
    for (int r = 0; r < kMaRpw; ++r) {
        if (rpos[r] < 0) continue;
        const int row = warp * kMaRpw + r;
        T* dst = static_cast<T*>(p.out) + (int64_t)(row0 + row / hc) * p.heads * p.vdim + (int64_t)rhead[r] * p.vdim;
        float ll = l[r];
        const float inv = p.sigm ? 1.f : ma_sink(p, rhead[r], m[r], ll) / ll;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int col = lane + 32 * i;
            float v = acc[r][i] * inv;
            if (p.out_rot) {                           // the partner column sits in the neighbouring lane (vdim is even)
                const float o = __shfl_xor_sync(0xffffffffu, v, 1);
                if (col < p.vdim) v = ma_unturn(p, row0 + row / hc, col, v, o);
            }
            if (p.gate && col < p.vdim) v *= ma_gate<T>(p, row0 + row / hc, rhead[r] * p.vdim + col);
            if (col < p.vdim) dst[col] = from_f32<T>(v);
        }
    }
}

template <typename T, int NV>
static int ma_launch(const MaskAttnParams& p, int ntiles, cudaStream_t st) {
    int hpg, hc, nchunk;
    hpg = p.heads / p.num_kv_heads;
    hc = hpg < kMaRows ? hpg : kMaRows;
    nchunk = (hpg + hc - 1) / hc;
    const size_t smem = ((size_t)kMaRows * p.dim + (size_t)kMaKeys * (p.dim + 1) + (size_t)kMaKeys * p.vdim) * sizeof(float);
    if (smem > 200 * 1024) return PA_ERR_UNSUPPORTED;
    cudaError_t e = cudaFuncSetAttribute(masked_attention_kernel<T, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    dim3 grid((unsigned)ntiles, (unsigned)(p.num_kv_heads * nchunk));
    masked_attention_kernel<T, NV><<<grid, kMaWarps * 32, smem, st>>>(p);
    PA_RETURN_LAUNCH_STATUS();
}

template <typename T>
static int ma_dispatch(const MaskAttnParams& p, int ntiles, cudaStream_t st) {
    const int nv = (p.vdim + 31) / 32;
    switch (nv) {
        case 1: return ma_launch<T, 1>(p, ntiles, st);
        case 2: return ma_launch<T, 2>(p, ntiles, st);
        case 3: return ma_launch<T, 3>(p, ntiles, st);
        case 4: return ma_launch<T, 4>(p, ntiles, st);
        case 5: case 6: return ma_launch<T, 6>(p, ntiles, st);
        case 7: case 8: return ma_launch<T, 8>(p, ntiles, st);
        default: return PA_ERR_UNSUPPORTED;
    }
}


// ---- single-token tiles (decode) ------------------------------------------------------------------------------------
// One CTA = one token x one key/value head; its R >= heads-per-kv-head rows are the query heads of the group.  Nothing is
// staged: each of the kMaDecWarps warps takes every kMaDecWarps-th run of 32 keys of the visible range, a lane reads ITS key's row with 16-byte
// loads straight into the dot products of every row (queries broadcast from shared memory), the warp does the online
// softmax, then lanes switch to value columns and read each key's value row coalesced.  The warps' (m, l, acc) are
// merged through shared memory.  Needs dim a multiple of the 16-byte vector and R <= 8 (else the tile kernel serves).
template <typename T> struct MaVec { static constexpr int N = 16 / sizeof(T); };

template <typename T>
__device__ __forceinline__ void ma_load16(const T* __restrict__ p, float (&f)[MaVec<T>::N]) {
    const uint4 v = ldg_stream_128(p);
    if (sizeof(T) == 4) {
        f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y); f[2] = __uint_as_float(v.z); f[3] = __uint_as_float(v.w);
    } else {
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            f[2 * i] = __uint_as_float(w[i] << 16);
            f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
}

// NV consecutive values of a row starting at element lane * NV, in one load where NV * sizeof(T) is 4, 8 or a multiple of 16
template <typename T, int NV>
__device__ __forceinline__ void ma_load_packed(const T* __restrict__ p, float (&f)[NV]) {
    constexpr int BYTES = NV * sizeof(T);
    if (BYTES % 16 == 0) {
#pragma unroll
        for (int c = 0; c < BYTES / 16; ++c) {
            float t[MaVec<T>::N];
            ma_load16<T>(p + c * MaVec<T>::N, t);
#pragma unroll
            for (int i = 0; i < MaVec<T>::N; ++i) f[c * MaVec<T>::N + i] = t[i];
        }
    } else if (BYTES == 8 && sizeof(T) == 2) {
        const uint2 v = ldg_stream_64(p);
        f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xffff0000u);
        f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xffff0000u);
    } else if (BYTES == 8) {
        const uint2 v = ldg_stream_64(p);
        f[0] = __uint_as_float(v.x); f[1] = __uint_as_float(v.y);
    } else if (BYTES == 4 && sizeof(T) == 2) {
        const uint32_t v = *reinterpret_cast<const uint32_t*>(p);
        f[0] = __uint_as_float(v << 16); f[1] = __uint_as_float(v & 0xffff0000u);
    } else {
#pragma unroll
        for (int i = 0; i < NV; ++i) f[i] = to_f32<T>(p[i]);
    }
}

// value column held in slot i of a lane: lane + 32 i, or (PACKED: vdim == 32 NV) lane * NV + i
template <int NV, bool PACKED>
__device__ __forceinline__ int ma_col(int lane, int i) { return PACKED ? lane * NV + i : lane + 32 * i; }

constexpr int kMaDecWarps = 16;   // a window of ~1000 keys leaves each warp two steps: the chain of dependent loads stays short

template <typename T, int R, int NV, bool PACKED>
__global__ void __launch_bounds__(kMaDecWarps * 32) masked_attention_decode_kernel(const MaskAttnParams p) {
    extern __shared__ float smem[];
    constexpr int VN = MaVec<T>::N;
    const int kd = p.dim;
    float* Qs = smem;                                   // [R][kd]
    float* Ps = Qs + R * kd;                            // [warps][R][2 + vdim]
    const int pstride = 2 + p.vdim;
    const int hpg = p.heads / p.num_kv_heads;
    const int* tile = p.tiles + 4 * blockIdx.x;
    const int row0 = tile[0], slot = tile[2], pos = tile[3];
    const int g = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const T* kp = static_cast<const T*>(p.k_pool);
    const T* vp = static_cast<const T*>(p.v_pool);
    for (int idx = threadIdx.x; idx < R * kd; idx += blockDim.x) {
        const int r = idx / kd, d = idx % kd;
        Qs[idx] = r < hpg ? to_f32<T>(static_cast<const T*>(p.q)[(int64_t)row0 * p.q_stride + p.q_off + (int64_t)(g * hpg + r) * kd + d]) : 0.f;
    }
    __syncthreads();
    float m[R], l[R], acc[R][NV], slope[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
        m[r] = -INFINITY;
        l[r] = 0.f;
        slope[r] = p.bias_kind == 1 && r < hpg ? p.bias[g * hpg + r] : 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) acc[r][i] = 0.f;
    }
    const int total = pos + 1;
    const MaSteps steps = ma_steps(p, ma_first_key(p, pos), total, kMaKeys);
    const int32_t* trow = p.table + ((int64_t)slot * p.num_kv_heads + g) * p.num_tiles;
    for (int sn = warp; sn < steps.count; sn += kMaDecWarps) {
        const int st = steps.step(sn);
        const int j = st * kMaKeys + lane;
        int prow = -1;                                  // pool row of this lane's key
        if (j < total && ma_visible(p, pos, j) && j / p.tile_size < p.num_tiles) {
            const int page = trow[j / p.tile_size];
            if (page >= 0 && page < p.total_pages) prow = page * p.tile_size + j % p.tile_size;
        }
        float s[R];
#pragma unroll
        for (int r = 0; r < R; ++r) s[r] = 0.f;
        if (prow >= 0) {
            const T* kr = kp + (int64_t)prow * kd;
#pragma unroll 8
            for (int d0 = 0; d0 < kd; d0 += VN) {
                float kv[VN];
                ma_load16<T>(kr + d0, kv);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const float* q = Qs + r * kd + d0;
#pragma unroll
                    for (int i = 0; i < VN; ++i) s[r] = fmaf(q[i], kv[i], s[r]);
                }
            }
        }
        const bool vis = prow >= 0;
        const float ks = vis && p.key_scale ? p.key_scale[prow] : 1.f;
        float w[R];
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const float v = vis && r < hpg ? ma_score(p, s[r] * ks, pos, j, g * hpg + r, slope[r]) : -INFINITY;
            if (p.sigm) {
                w[r] = v == -INFINITY ? 0.f : sigmoid_f32(v);
                continue;
            }
            const float n = fmaxf(m[r], warp_max(v));
            const float c = n == -INFINITY ? 1.f : expf(m[r] - n);
            w[r] = v == -INFINITY ? 0.f : expf(v - n);
            l[r] = l[r] * c + warp_sum(w[r]);
            m[r] = n;
#pragma unroll
            for (int i = 0; i < NV; ++i) acc[r][i] *= c;
        }
        const int nk = min(kMaKeys, total - st * kMaKeys);
#pragma unroll 8
        for (int jj = 0; jj < nk; ++jj) {
            const int pr = __shfl_sync(0xffffffffu, prow, jj);
            float v[NV];
#pragma unroll
            for (int i = 0; i < NV; ++i) v[i] = 0.f;
            if (pr >= 0) {
                const T* vr = vp + (int64_t)pr * p.vdim;
                if (PACKED) {
                    ma_load_packed<T, NV>(vr + lane * NV, v);
                } else {
#pragma unroll
                    for (int i = 0; i < NV; ++i) v[i] = lane + 32 * i < p.vdim ? to_f32<T>(vr[lane + 32 * i]) : 0.f;
                }
            }
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float wj = __shfl_sync(0xffffffffu, w[r], jj);
#pragma unroll
                for (int i = 0; i < NV; ++i) acc[r][i] = fmaf(wj, v[i], acc[r][i]);
            }
        }
    }
    // ---- the warps' partials -> shared memory, merged by warp r for row r
#pragma unroll
    for (int r = 0; r < R; ++r) {
        float* dst = Ps + ((int64_t)warp * R + r) * pstride;
        if (lane == 0) { dst[0] = m[r]; dst[1] = l[r]; }
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (ma_col<NV, PACKED>(lane, i) < p.vdim) dst[2 + ma_col<NV, PACKED>(lane, i)] = acc[r][i];
    }
    __syncthreads();
    for (int r = warp; r < R; r += kMaDecWarps) {
        if (r >= hpg) continue;
        float M = -INFINITY;
        for (int w = 0; w < kMaDecWarps; ++w) M = fmaxf(M, Ps[((int64_t)w * R + r) * pstride]);
        if (p.sink) M = fmaxf(M, p.sink[g * hpg + r]);
        if (p.sigm) M = 0.f;
        float L = p.sink ? expf(p.sink[g * hpg + r] - M) : 0.f, b[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) b[i] = 0.f;
        for (int w = 0; w < kMaDecWarps; ++w) {
            const float* pw = Ps + ((int64_t)w * R + r) * pstride;
            const float f = p.sigm ? 1.f : pw[0] == -INFINITY ? 0.f : expf(pw[0] - M);
            L = fmaf(f, pw[1], L);
#pragma unroll
            for (int i = 0; i < NV; ++i)
                if (ma_col<NV, PACKED>(lane, i) < p.vdim) b[i] = fmaf(f, pw[2 + ma_col<NV, PACKED>(lane, i)], b[i]);
        }
        T* dst = static_cast<T*>(p.out) + (int64_t)row0 * p.heads * p.vdim + (int64_t)(g * hpg + r) * p.vdim;
        const float inv = p.sigm ? 1.0f : 1.0f / L;
#pragma unroll
        for (int i = 0; i < NV; ++i) b[i] *= inv;
        if (p.out_rot) {          // the partner column: the neighbouring slot of this lane (packed pairs) or the neighbouring lane
            float o[NV];
#pragma unroll
            for (int i = 0; i < NV; ++i) o[i] = (PACKED && NV > 1) ? b[i ^ 1] : __shfl_xor_sync(0xffffffffu, b[i], 1);
#pragma unroll
            for (int i = 0; i < NV; ++i)
                if (ma_col<NV, PACKED>(lane, i) < p.vdim) b[i] = ma_unturn(p, row0, ma_col<NV, PACKED>(lane, i), b[i], o[i]);
        }
        if (p.gate) {
#pragma unroll
            for (int i = 0; i < NV; ++i)
                if (ma_col<NV, PACKED>(lane, i) < p.vdim) b[i] *= ma_gate<T>(p, row0, (g * hpg + r) * p.vdim + ma_col<NV, PACKED>(lane, i));
        }
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (ma_col<NV, PACKED>(lane, i) < p.vdim) dst[ma_col<NV, PACKED>(lane, i)] = from_f32<T>(b[i]);
    }
}

template <typename T, int R, int NV>
static int ma_decode_launch(const MaskAttnParams& p, int ntiles, cudaStream_t st) {
    const size_t smem = ((size_t)R * p.dim + (size_t)kMaDecWarps * R * (2 + p.vdim)) * sizeof(float);
    if (smem > 200 * 1024) return PA_ERR_UNSUPPORTED;
    // one load per lane and value row where the row is exactly 32 lanes x NV values and the pool is aligned for it
    const bool packed = p.vdim == 32 * NV && (uintptr_t)p.v_pool % 16 == 0 &&
                        ((NV * sizeof(T)) % 16 == 0 || NV * sizeof(T) == 8 || (NV * sizeof(T) == 4 && sizeof(T) == 2));
    auto kern = packed ? masked_attention_decode_kernel<T, R, NV, true> : masked_attention_decode_kernel<T, R, NV, false>;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    dim3 grid((unsigned)ntiles, (unsigned)p.num_kv_heads);
    kern<<<grid, kMaDecWarps * 32, smem, st>>>(p);
    PA_RETURN_LAUNCH_STATUS();
}

// PA_ERR_UNSUPPORTED: this shape stays on the tile kernel
template <typename T>
static int ma_decode_dispatch(const MaskAttnParams& p, int ntiles, cudaStream_t st) {
    const int hpg = p.heads / p.num_kv_heads, nv = (p.vdim + 31) / 32;
    if (p.dim % MaVec<T>::N || hpg > 8 || nv > 8) return PA_ERR_UNSUPPORTED;
    if ((uintptr_t)p.k_pool % 16) return PA_ERR_UNSUPPORTED;
    const int NVc = nv <= 1 ? 1 : nv <= 2 ? 2 : nv <= 4 ? 4 : 8;
#define PA_MA_DEC(RR)                                                   \
    switch (NVc) {                                                      \
        case 1: return ma_decode_launch<T, RR, 1>(p, ntiles, st);       \
        case 2: return ma_decode_launch<T, RR, 2>(p, ntiles, st);       \
        case 4: return ma_decode_launch<T, RR, 4>(p, ntiles, st);       \
        default: if (RR <= 4) return ma_decode_launch<T, (RR <= 4 ? RR : 4), 8>(p, ntiles, st); return PA_ERR_UNSUPPORTED; \
    }
    if (hpg <= 2) { PA_MA_DEC(2) }
    if (hpg <= 4) { PA_MA_DEC(4) }
    PA_MA_DEC(8)
#undef PA_MA_DEC
}

// ---- prompt portions on the tensor cores (bfloat16) -------------------------------------------------------------------
// One CTA = up to 64 consecutive tokens of one portion x ONE query head; 4 warps, warp w owns rows 16 w .. 16 w + 15:
// a flash-attention (mma.sync m16n8k16, bfloat16 operands, float accumulators) over staged key and value tiles of 64 keys,
// located through the page table and brought in with 16-byte cp.async copies into two buffers (the copies of step t + 1
// fly while step t is multiplied).  Only the key steps between the first key the tile's first token sees and its last
// token are visited; a warp skips steps none of its rows can see.  The dot products are raw q . k; scale, soft cap and
// distance bias are applied to the float score.  Scores, the running maximum, the exponentials and their sum are float;
// the weights enter the second product rounded to bfloat16, like every other matrix operand of this precision.
// DIM and VDIM are the PADDED sizes (32, 64 or 128): the real dim / vdim values (any multiple of 8) sit at the start of
// the columns and the rest is zero; 16-wide steps that are all padding are skipped.  A bias table of up to kMmBiasMax
// distances is staged (this head's column) in shared memory.  SIGM: sigmoid weights (no running maximum, no sum, no
// rescaling of the accumulators).  SHARED: the values are the key rows, so ONE staged tile serves both products.
constexpr int kMmRows = 64, kMmKeys = 64, kMmThreads = 128, kMmPad = 8, kMmStages = 2, kMmBiasMax = 4096;

__device__ __forceinline__ float ma_tanh(float x) {        // 1 - 2 / (e^{2x} + 1), relative error ~1e-6
    const float e = __expf(2.0f * x);
    return 1.0f - __fdividef(2.0f, e + 1.0f);
}

template <int DIM, int VDIM, bool SIGM, bool SHARED>
__global__ void __launch_bounds__(kMmThreads) masked_attention_mma_kernel(const MaskAttnParams p) {
    static_assert(!SHARED || DIM == VDIM, "values that are the keys have their size");
    constexpr int KS = DIM + kMmPad, VS = VDIM + kMmPad, NT = VDIM / 8, NST = kMmStages;
    extern __shared__ __align__(16) unsigned char mm_smem[];
    bf16_t* Qs = reinterpret_cast<bf16_t*>(mm_smem);         // [64][KS]
    bf16_t* Ks = Qs + kMmRows * KS;                           // [NST][64][KS]
    bf16_t* Vs = SHARED ? Ks : Ks + NST * kMmKeys * KS;       // [NST][64][VS]
    float* Bs = reinterpret_cast<float*>(Vs + NST * kMmKeys * VS);   // [bias_len] (bias_kind 2, bias_len <= kMmBiasMax)
    __shared__ int key_ok[NST][kMmKeys];
    __shared__ __align__(8) float key_sc[NST][kMmKeys];

    const int* tile = p.tiles + 4 * blockIdx.x;
    const int row0 = tile[0], ntok = tile[1], slot = tile[2], pos0 = tile[3];
    const int head = blockIdx.y, hpg = p.heads / p.num_kv_heads, g = head / hpg;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int rbase = warp * 16;
    const bool active = rbase < ntok;
    const bf16_t* kp = static_cast<const bf16_t*>(p.k_pool);
    const bf16_t* vp = static_cast<const bf16_t*>(p.v_pool);
    const int32_t* trow = p.table + ((int64_t)slot * p.num_kv_heads + g) * p.num_tiles;
    const int total = pos0 + ntok;
    const MaSteps steps = ma_steps(p, ma_first_key(p, pos0), total, kMmKeys);
    const int keep = p.mask_kind == 1 ? p.mask_keep : 0;
    const int dim = p.dim, vdim = p.vdim;
    const bool bias_smem = p.bias_kind == 2 && p.bias_len <= kMmBiasMax;

    for (int c = tid; c < kMmRows * (DIM / 8); c += kMmThreads) {
        const int r = c / (DIM / 8), cv = (c % (DIM / 8)) * 8;
        const bool ok = r < ntok && cv < dim;
        const bf16_t* src = static_cast<const bf16_t*>(p.q) + (ok ? (int64_t)(row0 + r) * p.q_stride + p.q_off + (int64_t)head * dim + cv : 0);
        cp_async_16(smem_u32(Qs + r * KS + cv), src, ok);
    }
    if (bias_smem)
        for (int d = tid; d < p.bias_len; d += kMmThreads) Bs[d] = p.bias[(int64_t)d * p.heads + head];
    auto pool_row = [&](int j) -> int64_t {
        if (j < total && j / p.tile_size < p.num_tiles) {
            const int page = trow[j / p.tile_size];
            if (page >= 0 && page < p.total_pages) return (int64_t)page * p.tile_size + j % p.tile_size;
        }
        return -1;
    };
    // two threads per key: ONE page look-up per thread and step; a thread copies every second 16-byte piece of its key's
    // row and of its value row
    auto load_tile = [&](int kt, int buf) {
        const int key = tid >> 1, q2 = tid & 1;
        const int64_t pr = pool_row(kt * kMmKeys + key);
        if (q2 == 0) {
            key_ok[buf][key] = pr >= 0;
            if (p.key_scale) cp_async_4(smem_u32(&key_sc[buf][key]), p.key_scale + (pr >= 0 ? pr : 0), pr >= 0);
        }
        bf16_t* kdst = Ks + (buf * kMmKeys + key) * KS;
        const bf16_t* ksrc = kp + (pr >= 0 ? pr * dim : 0);
#pragma unroll
        for (int i = 0; i < DIM / 16; ++i) {
            const int cv = (q2 + 2 * i) * 8;
            const bool ok = pr >= 0 && cv < dim;
            cp_async_16(smem_u32(kdst + cv), ok ? ksrc + cv : kp, ok);
        }
        if (SHARED) return;
        bf16_t* vdst = Vs + (buf * kMmKeys + key) * VS;
        const bf16_t* vsrc = vp + (pr >= 0 ? pr * vdim : 0);
#pragma unroll
        for (int i = 0; i < VDIM / 16; ++i) {
            const int cv = (q2 + 2 * i) * 8;
            const bool ok = pr >= 0 && cv < vdim;
            cp_async_16(smem_u32(vdst + cv), ok ? vsrc + cv : vp, ok);
        }
    };
#pragma unroll
    for (int t = 0; t < NST - 1; ++t) {
        if (t < steps.count) load_tile(steps.step(t), t);
        cp_async_commit();
    }

    float o[NT][4];
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int c = 0; c < 4; ++c) o[t][c] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    int rpos[2], rlo[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        rpos[i] = pos0 + rbase + (lane >> 2) + 8 * i;
        rlo[i] = ma_first_key(p, rpos[i]);
    }
    // the warp's rows together see keys [wlo, whi]
    const int wlo = ma_first_key(p, pos0 + rbase), whi = pos0 + min(rbase + 15, ntok - 1);
    const float slope = p.bias_kind == 1 ? p.bias[head] : 0.f;
    const float hscale = p.head_scale ? p.head_scale[head] : 1.f;
    const float hbias = p.head_bias ? p.head_bias[head] : 0.f;
    const float inv_cap = p.softcap > 0.f ? 1.0f / p.softcap : 0.f;
    constexpr float kLog2e = 1.4426950408889634f;

    for (int sn = 0; sn < steps.count; ++sn) {
        const int buf = sn % NST, c0 = steps.step(sn) * kMmKeys;
        if (sn + NST - 1 < steps.count) load_tile(steps.step(sn + NST - 1), (sn + NST - 1) % NST);
        cp_async_commit();
        cp_async_wait<NST - 1>();
        __syncthreads();
        if (active && ((c0 + kMmKeys - 1 >= wlo && c0 <= whi) || c0 < keep)) {
        float s[8][4];
#pragma unroll
        for (int t = 0; t < 8; ++t)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[t][c] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DIM; ks += 16) {
            if (ks >= dim) continue;                         // all padding
            uint32_t a[4];
            ldsm_x4(smem_u32(Qs + (rbase + (lane & 15)) * KS + ks + (lane >> 4) * 8), a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int np = 0; np < 4; ++np) {
                uint32_t b0, b1, b2, b3;
                ldsm_x4(smem_u32(Ks + (buf * kMmKeys + np * 16 + (lane & 7) + ((lane >> 4) << 3)) * KS + ks + ((lane >> 3) & 1) * 8),
                        b0, b1, b2, b3);
                mma_bf16_16816(s[2 * np], a, b0, b1);
                mma_bf16_16816(s[2 * np + 1], a, b2, b3);
            }
        }
        // ---- float scores -> weights (log2 domain)
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int t = 0; t < 8; ++t) {
            const int col = t * 8 + 2 * (lane & 3);
            const int2 okk = *reinterpret_cast<const int2*>(&key_ok[buf][col]);
            const float2 ksc = p.key_scale ? *reinterpret_cast<const float2*>(&key_sc[buf][col]) : make_float2(1.f, 1.f);
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int i = c >> 1, j = c0 + col + (c & 1);
                const bool vis = ((c & 1) ? okk.y : okk.x) && j <= rpos[i] && (j >= rlo[i] || j < keep);
                float v = s[t][c] * p.scale;
                if (p.key_scale) v *= (c & 1) ? ksc.y : ksc.x;
                if (p.head_scale) v *= hscale;
                if (p.softcap > 0.f) v = p.softcap * ma_tanh(v * inv_cap);
                if (p.bias_kind == 1) v -= slope * (float)(rpos[i] - j);
                else if (p.bias_kind == 2 && vis) {
                    const int dist = min(rpos[i] - j, p.bias_len - 1);
                    v += bias_smem ? Bs[dist] : p.bias[(int64_t)dist * p.heads + head];
                }
                if (SIGM) {
                    s[t][c] = vis ? __fdividef(1.0f, 1.0f + exp2f(-kLog2e * (v + hbias))) : 0.f;
                    continue;
                }
                s[t][c] = vis ? (v + hbias) * kLog2e : -INFINITY;
                mx[i] = fmaxf(mx[i], s[t][c]);
            }
        }
        if (!SIGM) {
        float ref[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
            mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
            const float mn = fmaxf(m[i], mx[i]);
            ref[i] = mn == -INFINITY ? 0.f : mn;
            const float corr = exp2f(m[i] - ref[i]);         // m = -inf: 0 (nothing accumulated yet)
            m[i] = mn;
            l[i] *= corr;
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                o[t][2 * i] *= corr;
                o[t][2 * i + 1] *= corr;
            }
        }
#pragma unroll
        for (int t = 0; t < 8; ++t)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                s[t][c] = exp2f(s[t][c] - ref[c >> 1]);
                l[c >> 1] += s[t][c];
            }
        }
        // ---- weighted sums
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t a[4];
            a[0] = pack_bf16x2(s[2 * kk][0], s[2 * kk][1]);
            a[1] = pack_bf16x2(s[2 * kk][2], s[2 * kk][3]);
            a[2] = pack_bf16x2(s[2 * kk + 1][0], s[2 * kk + 1][1]);
            a[3] = pack_bf16x2(s[2 * kk + 1][2], s[2 * kk + 1][3]);
#pragma unroll
            for (int np = 0; np < NT / 2; ++np) {
                if (np * 16 >= vdim) continue;               // all padding
                uint32_t b0, b1, b2, b3;
                ldsm_x4_trans(smem_u32(Vs + (buf * kMmKeys + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VS + np * 16 + (lane >> 4) * 8),
                              b0, b1, b2, b3);
                mma_bf16_16816(o[2 * np], a, b0, b1);
                mma_bf16_16816(o[2 * np + 1], a, b2, b3);
            }
        }
        }
        __syncthreads();                                     // this buffer is free for the copies of step kt + NST
    }
    cp_async_wait<0>();
    if (!active) return;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
        const int r = rbase + (lane >> 2) + 8 * i;
        if (r >= ntok) continue;
        float inv = SIGM ? 1.0f : 1.0f / l[i];
        if (!SIGM && p.sink) {                                        // the running maximum is in the log2 domain
            const float sk = p.sink[head] * kLog2e, mn = fmaxf(m[i], sk);
            const float corr = exp2f(m[i] - mn);
            inv = corr / (l[i] * corr + exp2f(sk - mn));
        }
        bf16_t* dst = static_cast<bf16_t*>(p.out) + (int64_t)(row0 + r) * p.heads * vdim + (int64_t)head * vdim + 2 * (lane & 3);
#pragma unroll
        for (int t = 0; t < NT; ++t) {
            if (t * 8 >= vdim) continue;
            float u = o[t][2 * i] * inv, v = o[t][2 * i + 1] * inv;
            if (p.out_rot) {                                 // a thread holds both columns of a pair
                const int col = t * 8 + 2 * (lane & 3);
                const float u0 = u;
                u = ma_unturn(p, row0 + r, col, u0, v);
                v = ma_unturn(p, row0 + r, col + 1, v, u0);
            }
            if (p.gate) {
                const int col = head * vdim + t * 8 + 2 * (lane & 3);
                u *= ma_gate<bf16_t>(p, row0 + r, col);
                v *= ma_gate<bf16_t>(p, row0 + r, col + 1);
            }
            *reinterpret_cast<uint32_t*>(dst + t * 8) = pack_bf16x2(u, v);
        }
    }
}

template <int DIM, int VDIM, bool SIGM, bool SHARED>
static int mm_launch(const MaskAttnParams& p, int ntiles, cudaStream_t st) {
    size_t smem = ((size_t)(kMmRows + kMmStages * kMmKeys) * (DIM + kMmPad) +
                   (SHARED ? 0 : (size_t)kMmStages * kMmKeys * (VDIM + kMmPad))) * sizeof(bf16_t);
    if (p.bias_kind == 2 && p.bias_len <= kMmBiasMax) smem += (size_t)p.bias_len * sizeof(float);
    auto kern = masked_attention_mma_kernel<DIM, VDIM, SIGM, SHARED>;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    dim3 grid((unsigned)ntiles, (unsigned)p.heads);
    kern<<<grid, kMmThreads, smem, st>>>(p);
    PA_RETURN_LAUNCH_STATUS();
}

static bool mm_shape_ok(int dim, int vdim) { return dim % 8 == 0 && dim <= 128 && vdim % 8 == 0 && vdim <= 128; }
static int mm_padded(int n) { return n <= 32 ? 32 : n <= 64 ? 64 : 128; }

static bool mm_operands_ok(const MaskAttnParams& p) {
    return mm_shape_ok(p.dim, p.vdim) && p.q_stride % 8 == 0 && p.q_off % 8 == 0 && (uintptr_t)p.q % 16 == 0 &&
           (uintptr_t)p.k_pool % 16 == 0 && (uintptr_t)p.v_pool % 16 == 0 && (uintptr_t)p.out % 4 == 0;
}

// PA_ERR_UNSUPPORTED: this shape or these pointers stay on the float kernel
static int mm_dispatch(const MaskAttnParams& p, int ntiles, cudaStream_t st) {
    if (!mm_operands_ok(p)) return PA_ERR_UNSUPPORTED;
    const int dp = mm_padded(p.dim), vp = mm_padded(p.vdim);
    if (p.k_pool == p.v_pool) {
#define PA_MM_CASE(D) if (dp == D) return p.sigm ? mm_launch<D, D, true, true>(p, ntiles, st) : mm_launch<D, D, false, true>(p, ntiles, st)
        PA_MM_CASE(32); PA_MM_CASE(64); PA_MM_CASE(128);
#undef PA_MM_CASE
        return PA_ERR_UNSUPPORTED;
    }
#define PA_MM_CASE(D, V) if (dp == D && vp == V) return p.sigm ? mm_launch<D, V, true, false>(p, ntiles, st) : mm_launch<D, V, false, false>(p, ntiles, st)
    PA_MM_CASE(32, 32); PA_MM_CASE(32, 64); PA_MM_CASE(32, 128);
    PA_MM_CASE(64, 32); PA_MM_CASE(64, 64); PA_MM_CASE(64, 128);
    PA_MM_CASE(128, 32); PA_MM_CASE(128, 64); PA_MM_CASE(128, 128);
#undef PA_MM_CASE
    return PA_ERR_UNSUPPORTED;
}

// ---- decoded tokens on the tensor cores (bfloat16) ---------------------------------------------------------------------
// One CTA = one token x one key/value head x up to 16 of its query heads, which are the ROWS of the products.  The staged
// tiles are those of the portion kernel (64 keys, 16-byte cp.async copies, a ring of three or five buffers); the four warps split the 64
// keys of a step, 16 each, keep a running (m, l, o) of their own and meet in shared memory at the end.  Every cached row is
// read once, in whole lines, whatever the number of heads; for batches with at least one CTA per SM.
constexpr int kMdRows = 16;
constexpr int md_stages(bool shared) { return shared ? 5 : 3; }     // two resident CTAs per SM at 128-wide heads

template <int DIM, int VDIM, bool SHARED>
__global__ void __launch_bounds__(kMmThreads) masked_attention_mma_decode_kernel(const MaskAttnParams p) {
    static_assert(!SHARED || DIM == VDIM, "values that are the keys have their size");
    constexpr int KS = DIM + kMmPad, VS = VDIM + kMmPad, NT = VDIM / 8, NST = md_stages(SHARED), OS = VDIM + 4;
    extern __shared__ __align__(16) unsigned char mm_smem[];
    bf16_t* Qs = reinterpret_cast<bf16_t*>(mm_smem);         // [16][KS]
    bf16_t* Ks = Qs + kMdRows * KS;                           // [NST][64][KS]
    bf16_t* Vs = SHARED ? Ks : Ks + NST * kMmKeys * KS;       // [NST][64][VS]
    float* Os = reinterpret_cast<float*>(Ks);                 // [4][16][OS], over the tiles once they are consumed
    __shared__ int key_ok[NST][kMmKeys];
    __shared__ __align__(8) float key_sc[NST][kMmKeys];
    __shared__ float ms[4][kMdRows], ls[4][kMdRows];

    const int hpg = p.heads / p.num_kv_heads, nchunk = (hpg + kMdRows - 1) / kMdRows;
    const int* tile = p.tiles + 4 * blockIdx.x;
    const int row0 = tile[0], slot = tile[2], pos = tile[3];
    const int g = blockIdx.y / nchunk, hbase = g * hpg + blockIdx.y % nchunk * kMdRows;
    const int nrow = min(kMdRows, (g + 1) * hpg - hbase);     // query heads of this CTA
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bf16_t* kp = static_cast<const bf16_t*>(p.k_pool);
    const bf16_t* vp = static_cast<const bf16_t*>(p.v_pool);
    const int32_t* trow = p.table + ((int64_t)slot * p.num_kv_heads + g) * p.num_tiles;
    const int total = pos + 1, dim = p.dim, vdim = p.vdim;
    const MaSteps steps = ma_steps(p, ma_first_key(p, pos), total, kMmKeys);

    for (int c = tid; c < kMdRows * (DIM / 8); c += kMmThreads) {
        const int r = c / (DIM / 8), cv = (c % (DIM / 8)) * 8;
        const bool ok = r < nrow && cv < dim;
        const bf16_t* src = static_cast<const bf16_t*>(p.q) + (ok ? (int64_t)row0 * p.q_stride + p.q_off + (int64_t)(hbase + r) * dim + cv : 0);
        cp_async_16(smem_u32(Qs + r * KS + cv), src, ok);
    }
    // two threads per key; the page of a step's key is looked up one step before its copies are issued
    const int key = tid >> 1, q2 = tid & 1;
    auto look_up = [&](int sn) -> int64_t {
        if (sn >= steps.count) return -1;
        const int j = steps.step(sn) * kMmKeys + key;
        if (j < total && ma_visible(p, pos, j) && j / p.tile_size < p.num_tiles) {
            const int page = trow[j / p.tile_size];
            if (page >= 0 && page < p.total_pages) return (int64_t)page * p.tile_size + j % p.tile_size;
        }
        return -1;
    };
    auto load_tile = [&](int64_t pr, int buf) {
        if (q2 == 0) {
            key_ok[buf][key] = pr >= 0;
            if (p.key_scale) cp_async_4(smem_u32(&key_sc[buf][key]), p.key_scale + (pr >= 0 ? pr : 0), pr >= 0);
        }
        bf16_t* kdst = Ks + (buf * kMmKeys + key) * KS;
        const bf16_t* ksrc = kp + (pr >= 0 ? pr * dim : 0);
#pragma unroll
        for (int i = 0; i < DIM / 16; ++i) {
            const int cv = (q2 + 2 * i) * 8;
            const bool ok = pr >= 0 && cv < dim;
            cp_async_16(smem_u32(kdst + cv), ok ? ksrc + cv : kp, ok);
        }
        if (SHARED) return;
        bf16_t* vdst = Vs + (buf * kMmKeys + key) * VS;
        const bf16_t* vsrc = vp + (pr >= 0 ? pr * vdim : 0);
#pragma unroll
        for (int i = 0; i < VDIM / 16; ++i) {
            const int cv = (q2 + 2 * i) * 8;
            const bool ok = pr >= 0 && cv < vdim;
            cp_async_16(smem_u32(vdst + cv), ok ? vsrc + cv : vp, ok);
        }
    };
#pragma unroll
    for (int t = 0; t < NST - 1; ++t) {
        if (t < steps.count) load_tile(look_up(t), t);
        cp_async_commit();
    }
    int64_t ahead = look_up(NST - 1);

    float o[NT][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int c = 0; c < 4; ++c) o[t][c] = 0.f;
    const int r0 = lane >> 2;                                 // this thread's rows: r0 and r0 + 8
    const float inv_cap = p.softcap > 0.f ? 1.0f / p.softcap : 0.f;
    float slope[2], hfac[2], hbias[2];                        // of the two rows' heads
    const float* btab[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int h = hbase + min(r0 + 8 * i, nrow - 1);
        slope[i] = p.bias_kind == 1 ? p.bias[h] : 0.f;
        hfac[i] = p.scale * (p.head_scale ? p.head_scale[h] : 1.f);
        hbias[i] = p.head_bias ? p.head_bias[h] : 0.f;
        btab[i] = p.bias_kind == 2 ? p.bias + h : nullptr;
    }

    for (int sn = 0; sn < steps.count; ++sn) {
        const int buf = sn % NST, c0 = steps.step(sn) * kMmKeys;
        if (sn + NST - 1 < steps.count) load_tile(ahead, (sn + NST - 1) % NST);
        cp_async_commit();
        ahead = look_up(sn + NST);
        cp_async_wait<NST - 1>();
        __syncthreads();
        float s[2][4];
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int c = 0; c < 4; ++c) s[t][c] = 0.f;
        const bf16_t* kw = Ks + (buf * kMmKeys + warp * 16) * KS;
#pragma unroll
        for (int ks = 0; ks < DIM; ks += 16) {
            if (ks >= dim) continue;                         // all padding
            uint32_t a[4], b0, b1, b2, b3;
            ldsm_x4(smem_u32(Qs + (lane & 15) * KS + ks + (lane >> 4) * 8), a[0], a[1], a[2], a[3]);
            ldsm_x4(smem_u32(kw + ((lane & 7) + ((lane >> 4) << 3)) * KS + ks + ((lane >> 3) & 1) * 8), b0, b1, b2, b3);
            mma_bf16_16816(s[0], a, b0, b1);
            mma_bf16_16816(s[1], a, b2, b3);
        }
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int t = 0; t < 2; ++t) {
            const int col = warp * 16 + t * 8 + 2 * (lane & 3);
            const int2 okk = *reinterpret_cast<const int2*>(&key_ok[buf][col]);
            const float2 ksc = p.key_scale ? *reinterpret_cast<const float2*>(&key_sc[buf][col]) : make_float2(1.f, 1.f);
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                const int i = c >> 1, dist = pos - (c0 + col + (c & 1));
                const bool vis = ((c & 1) ? okk.y : okk.x) && r0 + 8 * i < nrow;
                float v = s[t][c] * ((c & 1) ? ksc.y : ksc.x) * hfac[i];
                if (p.softcap > 0.f) v = p.softcap * ma_tanh(v * inv_cap);
                if (p.bias_kind == 1) v -= slope[i] * (float)dist;
                else if (p.bias_kind == 2) v += btab[i][(int64_t)min(max(dist, 0), p.bias_len - 1) * p.heads];
                s[t][c] = vis ? v + hbias[i] : -INFINITY;
                mx[i] = fmaxf(mx[i], s[t][c]);
            }
        }
        if (p.sigm) {
#pragma unroll
            for (int t = 0; t < 2; ++t)
#pragma unroll
                for (int c = 0; c < 4; ++c) s[t][c] = s[t][c] == -INFINITY ? 0.f : __fdividef(1.0f, 1.0f + __expf(-s[t][c]));
        } else {
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
                mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
                const float mn = fmaxf(m[i], mx[i]), ref = mn == -INFINITY ? 0.f : mn;
                const float corr = __expf(m[i] - ref);       // m = -inf: 0 (nothing accumulated yet)
                m[i] = mn;
                l[i] *= corr;
#pragma unroll
                for (int t = 0; t < NT; ++t) {
                    o[t][2 * i] *= corr;
                    o[t][2 * i + 1] *= corr;
                }
#pragma unroll
                for (int t = 0; t < 2; ++t)
#pragma unroll
                    for (int c = 2 * i; c < 2 * i + 2; ++c) {
                        s[t][c] = __expf(s[t][c] - ref);
                        l[i] += s[t][c];
                    }
            }
        }
        uint32_t a[4] = {pack_bf16x2(s[0][0], s[0][1]), pack_bf16x2(s[0][2], s[0][3]), pack_bf16x2(s[1][0], s[1][1]), pack_bf16x2(s[1][2], s[1][3])};
        const bf16_t* vw = Vs + (buf * kMmKeys + warp * 16) * VS;
#pragma unroll
        for (int np = 0; np < NT / 2; ++np) {
            if (np * 16 >= vdim) continue;                   // all padding
            uint32_t b0, b1, b2, b3;
            ldsm_x4_trans(smem_u32(vw + ((lane & 7) + ((lane >> 3) & 1) * 8) * VS + np * 16 + (lane >> 4) * 8), b0, b1, b2, b3);
            mma_bf16_16816(o[2 * np], a, b0, b1);
            mma_bf16_16816(o[2 * np + 1], a, b2, b3);
        }
        __syncthreads();                                     // this buffer is free for the copies of step sn + NST
    }
    cp_async_wait<0>();
    __syncthreads();
    // ---- the warps' partial results -> shared memory
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
        if ((lane & 3) == 0) { ms[warp][r0 + 8 * i] = m[i]; ls[warp][r0 + 8 * i] = l[i]; }
        float* dst = Os + (warp * kMdRows + r0 + 8 * i) * OS + 2 * (lane & 3);
#pragma unroll
        for (int t = 0; t < NT; ++t) *reinterpret_cast<float2*>(dst + t * 8) = make_float2(o[t][2 * i], o[t][2 * i + 1]);
    }
    __syncthreads();
    for (int idx = tid; idx < nrow * (vdim >> 1); idx += kMmThreads) {
        const int r = idx / (vdim >> 1), col = idx % (vdim >> 1) * 2;
        float f[4], inv = 1.f;
        if (p.sigm) {
            f[0] = f[1] = f[2] = f[3] = 1.f;
        } else {
            float M = fmaxf(fmaxf(ms[0][r], ms[1][r]), fmaxf(ms[2][r], ms[3][r]));
            if (p.sink) M = fmaxf(M, p.sink[hbase + r]);
            float L = p.sink ? expf(p.sink[hbase + r] - M) : 0.f;
#pragma unroll
            for (int w = 0; w < 4; ++w) {
                f[w] = ms[w][r] == -INFINITY ? 0.f : expf(ms[w][r] - M);
                L = fmaf(f[w], ls[w][r], L);
            }
            inv = 1.0f / L;
        }
        float u = 0.f, v = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float2 ov = *reinterpret_cast<const float2*>(Os + (w * kMdRows + r) * OS + col);
            u = fmaf(f[w], ov.x, u);
            v = fmaf(f[w], ov.y, v);
        }
        u *= inv;
        v *= inv;
        if (p.out_rot) {
            const float u0 = u;
            u = ma_unturn(p, row0, col, u0, v);
            v = ma_unturn(p, row0, col + 1, v, u0);
        }
        const int64_t oc = (int64_t)(hbase + r) * vdim + col;
        if (p.gate) {
            u *= ma_gate<bf16_t>(p, row0, (int)oc);
            v *= ma_gate<bf16_t>(p, row0, (int)oc + 1);
        }
        *reinterpret_cast<uint32_t*>(static_cast<bf16_t*>(p.out) + (int64_t)row0 * p.heads * vdim + oc) = pack_bf16x2(u, v);
    }
}

template <int DIM, int VDIM, bool SHARED>
static int md_launch(const MaskAttnParams& p, int ntiles, cudaStream_t st) {
    const size_t tiles = ((size_t)md_stages(SHARED) * kMmKeys * (DIM + kMmPad) + (SHARED ? 0 : (size_t)md_stages(SHARED) * kMmKeys * (VDIM + kMmPad))) * sizeof(bf16_t);
    const size_t merge = (size_t)4 * kMdRows * (VDIM + 4) * sizeof(float);
    const size_t smem = (size_t)kMdRows * (DIM + kMmPad) * sizeof(bf16_t) + (tiles > merge ? tiles : merge);
    auto kern = masked_attention_mma_decode_kernel<DIM, VDIM, SHARED>;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    const int hpg = p.heads / p.num_kv_heads;
    dim3 grid((unsigned)ntiles, (unsigned)(p.num_kv_heads * ((hpg + kMdRows - 1) / kMdRows)));
    kern<<<grid, kMmThreads, smem, st>>>(p);
    PA_RETURN_LAUNCH_STATUS();
}

// PA_ERR_UNSUPPORTED: this shape or these pointers stay on the streaming kernel
static int md_dispatch(const MaskAttnParams& p, int ntiles, cudaStream_t st) {
    if (!mm_operands_ok(p)) return PA_ERR_UNSUPPORTED;
    const int dp = mm_padded(p.dim), vp = mm_padded(p.vdim);
    if (p.k_pool == p.v_pool) {
#define PA_MD_CASE(D) if (dp == D) return md_launch<D, D, true>(p, ntiles, st)
        PA_MD_CASE(32); PA_MD_CASE(64); PA_MD_CASE(128);
#undef PA_MD_CASE
        return PA_ERR_UNSUPPORTED;
    }
#define PA_MD_CASE(D, V) if (dp == D && vp == V) return md_launch<D, V, false>(p, ntiles, st)
    PA_MD_CASE(32, 32); PA_MD_CASE(32, 64); PA_MD_CASE(32, 128);
    PA_MD_CASE(64, 32); PA_MD_CASE(64, 64); PA_MD_CASE(64, 128);
    PA_MD_CASE(128, 32); PA_MD_CASE(128, 64); PA_MD_CASE(128, 128);
#undef PA_MD_CASE
    return PA_ERR_UNSUPPORTED;
}

}  // namespace pa

using namespace pa;

PA_API int pa_masked_attention_tile_tokens(int heads, int kv_heads) {
    if (heads <= 0 || kv_heads <= 0 || heads % kv_heads) return 0;
    const int hpg = heads / kv_heads;
    return kMaRows / (hpg < kMaRows ? hpg : kMaRows);
}

PA_API int pa_masked_attention(const void* d_q, int64_t q_stride, int q_off, const void* d_k_pool, const void* d_v_pool,
                               const int32_t* d_table, int num_slots, int num_kv_heads, int num_tiles, int total_pages,
                               int tile_size, const int32_t* d_q_tiles, int num_q_tiles, int heads, int dim, int vdim,
                               float scale, float softcap, int mask_kind, int mask_size, int bias_kind,
                               const float* d_bias, int bias_len, void* d_out, int elem, int tile_kind,
                               pa_stream_t stream) {
    return pa_masked_attention_sink(d_q, q_stride, q_off, d_k_pool, d_v_pool, d_table, num_slots, num_kv_heads, num_tiles,
                                    total_pages, tile_size, d_q_tiles, num_q_tiles, heads, dim, vdim, scale, softcap,
                                    mask_kind, mask_size, 0, bias_kind, d_bias, bias_len, nullptr, nullptr, nullptr, d_out,
                                    elem, tile_kind, stream);
}

PA_API int pa_masked_attention_sink(const void* d_q, int64_t q_stride, int q_off, const void* d_k_pool, const void* d_v_pool,
                                    const int32_t* d_table, int num_slots, int num_kv_heads, int num_tiles, int total_pages,
                                    int tile_size, const int32_t* d_q_tiles, int num_q_tiles, int heads, int dim, int vdim,
                                    float scale, float softcap, int mask_kind, int mask_size, int mask_keep, int bias_kind,
                                    const float* d_bias, int bias_len, const float* d_head_scale, const float* d_sink,
                                    const float* d_out_rot, void* d_out, int elem, int tile_kind, pa_stream_t stream) {
    return pa_masked_attention_gated(d_q, q_stride, q_off, d_k_pool, d_v_pool, d_table, num_slots, num_kv_heads, num_tiles,
                                     total_pages, tile_size, d_q_tiles, num_q_tiles, heads, dim, vdim, scale, softcap,
                                     mask_kind, mask_size, mask_keep, bias_kind, d_bias, bias_len, d_head_scale, d_sink,
                                     d_out_rot, nullptr, 0, nullptr, nullptr, 0, 0, d_out, elem, tile_kind, stream);
}

PA_API int pa_masked_attention_gated(const void* d_q, int64_t q_stride, int q_off, const void* d_k_pool, const void* d_v_pool,
                                     const int32_t* d_table, int num_slots, int num_kv_heads, int num_tiles, int total_pages,
                                     int tile_size, const int32_t* d_q_tiles, int num_q_tiles, int heads, int dim, int vdim,
                                     float scale, float softcap, int mask_kind, int mask_size, int mask_keep, int bias_kind,
                                     const float* d_bias, int bias_len, const float* d_head_scale, const float* d_sink,
                                     const float* d_out_rot, const float* d_key_scale, int sigmoid_weights,
                                     const float* d_head_bias, const void* d_gate, int64_t gate_stride, int gate_off,
                                     void* d_out, int elem, int tile_kind, pa_stream_t stream) {
    PA_CHECK_ARG((sigmoid_weights == 0 || sigmoid_weights == 1) && !(sigmoid_weights && d_sink) && (d_k_pool != d_v_pool || dim == vdim));
    PA_CHECK_ARG(mask_keep >= 0 && (mask_keep == 0 || mask_kind == 1) && (!d_out_rot || vdim % 2 == 0));
    PA_CHECK_ARG(d_q && d_k_pool && d_v_pool && d_table && d_q_tiles && d_out && num_q_tiles >= 0);
    PA_CHECK_ARG(num_slots > 0 && num_kv_heads > 0 && num_tiles > 0 && total_pages > 0 && tile_size > 0);
    PA_CHECK_ARG(heads > 0 && heads % num_kv_heads == 0 && dim > 0 && vdim > 0 && softcap >= 0.f);
    PA_CHECK_ARG(mask_kind >= 0 && mask_kind <= 2 && (mask_kind == 0 || mask_size > 0));
    PA_CHECK_ARG(bias_kind >= 0 && bias_kind <= 2 && (bias_kind == 0 || d_bias) && (bias_kind != 2 || bias_len > 0));
    if (num_q_tiles == 0) return PA_OK;
    MaskAttnParams p;
    p.q = d_q; p.q_stride = q_stride; p.q_off = q_off; p.k_pool = d_k_pool; p.v_pool = d_v_pool; p.table = d_table;
    p.num_slots = num_slots; p.num_kv_heads = num_kv_heads; p.num_tiles = num_tiles; p.total_pages = total_pages;
    p.tile_size = tile_size; p.tiles = d_q_tiles; p.heads = heads; p.dim = dim; p.vdim = vdim; p.scale = scale;
    p.softcap = softcap; p.mask_kind = mask_kind; p.mask_size = mask_size; p.bias_kind = bias_kind; p.bias = d_bias;
    p.bias_len = bias_len; p.out = d_out;
    p.head_scale = d_head_scale; p.sink = d_sink; p.mask_keep = mask_keep; p.out_rot = d_out_rot;
    p.sigm = sigmoid_weights; p.key_scale = d_key_scale; p.head_bias = d_head_bias; p.gate = d_gate;
    p.gate_stride = gate_stride; p.gate_off = gate_off;
    if (elem != 4 && elem != 2) return PA_ERR_UNSUPPORTED;
    if (tile_kind == 2) {       // on the tensor cores: tiles of up to pa_masked_attention_mma_tile_tokens tokens
        if (elem != 2) return PA_ERR_UNSUPPORTED;
        return mm_dispatch(p, num_q_tiles, as_stream(stream));
    }
    if (tile_kind == 3)         // every tile is one token: the heads of a kv head as rows on the tensor cores
        return elem == 2 ? md_dispatch(p, num_q_tiles, as_stream(stream)) : PA_ERR_UNSUPPORTED;
    if (tile_kind == 1) {       // every tile is one token: the streaming kernel, where it serves the shape
        const int st = elem == 4 ? ma_decode_dispatch<float>(p, num_q_tiles, as_stream(stream))
                                 : ma_decode_dispatch<bf16_t>(p, num_q_tiles, as_stream(stream));
        if (st != PA_ERR_UNSUPPORTED) return st;
    }
    if (elem == 4) return ma_dispatch<float>(p, num_q_tiles, as_stream(stream));
    return ma_dispatch<bf16_t>(p, num_q_tiles, as_stream(stream));
}

PA_API int pa_rope_kv_append(void* d_src, int64_t src_stride, int q_off, int k_off, int v_off, int heads, int kv_heads,
                             int dim, int vdim, int rot_dims, const float* d_rope, const float* d_value_rope,
                             void* d_k_pool, void* d_v_pool, const int32_t* d_table, int num_slots, int num_tiles,
                             int total_pages, int tile_size, const int32_t* d_row_slot, const int32_t* d_row_pos, int rows,
                             int elem, pa_stream_t stream) {
    PA_CHECK_ARG(d_src && rows >= 0 && heads > 0 && kv_heads > 0 && dim > 0 && vdim > 0);
    PA_CHECK_ARG(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim && (rot_dims == 0 || d_rope));
    PA_CHECK_ARG(!d_value_rope || vdim % 2 == 0);
    PA_CHECK_ARG(!d_k_pool || (d_v_pool && d_table && d_row_slot && d_row_pos && num_slots > 0 && num_tiles > 0 &&
                               total_pages > 0 && tile_size > 0));
    if (rows == 0) return PA_OK;
    const int64_t threads = (int64_t)rows * (heads + (d_k_pool ? kv_heads : 0)) * 32;
    PA_DISPATCH_ELEM(elem, rope_kv_append_kernel<T><<<(unsigned)((threads + 255) / 256), 256, 0, as_stream(stream)>>>(
                               static_cast<T*>(d_src), src_stride, q_off, k_off, v_off, heads, kv_heads, dim, vdim, rot_dims,
                               rot_dims ? d_rope : nullptr, d_value_rope, static_cast<T*>(d_k_pool),
                               static_cast<T*>(d_v_pool), d_table, num_slots, num_tiles, total_pages, tile_size, d_row_slot,
                               d_row_pos, rows));
    PA_RETURN_LAUNCH_STATUS();
}

PA_API int pa_qk_norm_kv_append(void* d_src, int64_t src_stride, int q_off, int k_off, int v_off, int heads, int kv_heads,
                                int dim, int vdim, const float* d_q_gain, const float* d_k_gain, float eps, void* d_k_pool,
                                void* d_v_pool, float* d_key_scale, const int32_t* d_table, int num_slots, int num_tiles,
                                int total_pages, int tile_size, const int32_t* d_row_slot, const int32_t* d_row_pos,
                                int rows, int elem, pa_stream_t stream) {
    PA_CHECK_ARG(d_src && rows >= 0 && heads > 0 && kv_heads > 0 && dim > 0 && d_q_gain && (d_k_gain || d_key_scale));
    PA_CHECK_ARG(d_k_pool && d_table && d_row_slot && d_row_pos && num_slots > 0 && num_tiles > 0 && total_pages > 0);
    PA_CHECK_ARG(tile_size > 0 && d_v_pool != d_k_pool && (!d_v_pool || vdim > 0));
    if (rows == 0) return PA_OK;
    const int64_t threads = (int64_t)rows * (heads + kv_heads) * 32;
    PA_DISPATCH_ELEM(elem, qk_norm_kv_append_kernel<T><<<(unsigned)((threads + 255) / 256), 256, 0, as_stream(stream)>>>(
                               static_cast<T*>(d_src), src_stride, q_off, k_off, v_off, heads, kv_heads, dim, vdim, d_q_gain,
                               d_k_gain, eps, static_cast<T*>(d_k_pool), static_cast<T*>(d_v_pool), d_key_scale, d_table,
                               num_slots, num_tiles, total_pages, tile_size, d_row_slot, d_row_pos, rows));
    PA_RETURN_LAUNCH_STATUS();
}

PA_API int pa_conv_rope_norm_append(const void* d_in, int64_t in_stride, int in_off, int heads, int kv_heads, int dim, int vdim,
                                    int taps, const float* d_weight, float* d_state, int rot_dims, const float* d_rope,
                                    int norm, float eps, void* d_q_out, int64_t q_out_stride, void* d_k_pool, void* d_v_pool,
                                    const int32_t* d_table, int num_slots, int num_tiles, int total_pages, int tile_size,
                                    const int32_t* d_items, int num_items, int item_tokens, int elem, pa_stream_t stream) {
    PA_CHECK_ARG(d_in && d_q_out && d_items && num_items >= 0 && heads > 0 && kv_heads > 0 && dim > 0 && vdim > 0 && num_slots > 0);
    PA_CHECK_ARG(rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim && (rot_dims == 0 || d_rope) && (norm == 0 || norm == 1));
    PA_CHECK_ARG(!d_weight || (taps >= 1 && taps <= kCaMaxTaps && (taps == 1 || d_state) && item_tokens >= taps - 1));
    PA_CHECK_ARG((d_k_pool != nullptr) == (d_v_pool != nullptr) && d_q_out != d_in);
    PA_CHECK_ARG(!d_k_pool || (d_table && num_tiles > 0 && total_pages > 0 && tile_size > 0));
    if (num_items == 0) return PA_OK;
    ConvAppendParams p;
    p.in = d_in; p.in_stride = in_stride; p.in_off = in_off; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim;
    p.channels = heads * dim + (d_k_pool ? kv_heads * (dim + vdim) : 0);
    p.rot_dims = rot_dims; p.taps = taps; p.w = d_weight; p.state = d_state; p.rope = d_rope; p.norm = norm; p.eps = eps;
    p.q_out = d_q_out; p.q_out_stride = q_out_stride; p.k_pool = d_k_pool; p.v_pool = d_v_pool; p.table = d_table;
    p.num_slots = num_slots; p.num_tiles = num_tiles; p.total_pages = total_pages; p.tile_size = tile_size;
    p.items = d_items; p.num_items = num_items;
    const uintptr_t two = 2 * (uintptr_t)(elem == 2 ? 2 : 4);
    p.pairs = dim % 2 == 0 && vdim % 2 == 0 && in_stride % 2 == 0 && in_off % 2 == 0 && q_out_stride % 2 == 0 &&
              ((uintptr_t)d_in | (uintptr_t)d_q_out | (uintptr_t)d_k_pool | (uintptr_t)d_v_pool) % two == 0;
    // the vector form: columns in words of four or eight, 32-bit unit numbers
    auto words = [&](int k) {
        const uintptr_t bytes = (uintptr_t)(k * (elem == 2 ? 2 : 4) < 16 ? k * 2 : 16);
        return dim % k == 0 && vdim % k == 0 && in_stride % k == 0 && in_off % k == 0 && q_out_stride % k == 0 &&
               ((uintptr_t)d_in | (uintptr_t)d_q_out | (uintptr_t)d_k_pool | (uintptr_t)d_v_pool) % bytes == 0;
    };
    const bool floats = ((uintptr_t)d_weight | (uintptr_t)d_state | (uintptr_t)d_rope) % 16 == 0 && rot_dims % 4 == 0;
    const bool small = (int64_t)num_items * (heads + 2 * kv_heads) < (1 << 26) && in_stride < (1 << 30);
    p.words = !floats || !small ? 0 : words(8) ? 8 : words(4) ? 4 : 0;
    if (elem == 4) return ca_dispatch<float>(p, as_stream(stream));
    if (elem == 2) return ca_dispatch<bf16_t>(p, as_stream(stream));
    return PA_ERR_UNSUPPORTED;
}

PA_API int pa_masked_attention_mma_tile_tokens(int dim, int vdim, int elem) {
    return elem == 2 && mm_shape_ok(dim, vdim) ? kMmRows : 0;
}

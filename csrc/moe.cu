// Mixture-of-experts feed-forwards (models/deluvik.py, models/tobadra.py): every token uses the `top` experts with the largest router
// logits, weighted by the softmax over those, and `pieces` experts that all tokens share (weight one).  Or (MoePlanArgs::outputs) scores
// are the softmax over all outputs; a correction joins them for the choice only, which keeps to the groups of neighbours with the
// largest best score; outputs past the experts stand for the token's own row; the shared experts have a gate per token.
//
//   moe_topk_kernel    router logits -> expert numbers and weights of every token, one warp per token.
//   moe_plan_kernel    (moe_plan_small_kernel for a few pairs) one block: orders the (token, expert) pairs by expert and cuts every expert's rows into tiles.  Ticks of few
//                      tokens choose their experts in here, too.  The place of a row among its expert's is arbitrary; its values are not.
//   moe_rows_kernel    few rows: gated up projection / down projection of every tile (up to 8 rows), weights streamed as in
//                      linear_rows.cu: a warp owns 16 weight rows and a share of K in its own slots of a ring.
//   moe_plain_kernel   the same on CUDA cores (fp32 models, widths the ring has no room for).
//   moe_gather_kernel  input rows in the order of the list, for the tensor-core tiles of moe_tc.cu.
//
// The weighted sum over a token's experts is part of join_kernel (join.cu).
// Reference parity: the reference has dense feed-forwards only (no counterpart).
#include "moe.cuh"

// Mirrored by tilerl_b200/ops/cuda_blocks.py::MoePlan, field by field.
struct MoePlanArgs {
  const float* z;                      // [T, ldz] router products
  const float* bias;                   // [experts]
  int* ids;                            // [T, slots]
  float* weight;                       // [T, slots]
  int* place;                          // [T, slots]: row of the pair in the list
  int* token;                          // [T * slots]: token of a row
  MoeItem* items;
  int* n_items;
  int T, ldz, experts, top, pieces, tile, max_items;
  // grouped choice (outputs 0: none): bias is the correction; gate_col: column of z with the shared experts' gate (-1: none)
  int outputs, groups, keep, gate_col;
  float scale;
};

namespace {

constexpr int MP_THREADS = 1024, MP_MAXE = 2048;

// Chooses one token's experts (a warp).  Not-a-number counts as minus infinity, so the choice is always `top` different experts.
__device__ __forceinline__ void choose_experts(const MoePlanArgs& a, int t) {
  const int lane = threadIdx.x & 31, slots = a.top + a.pieces;
  const float* z = a.z + (size_t)t * a.ldz;
  float first = 0.f, sum = 0.f, last = INFINITY;
  int last_id = -1;
  for (int j = 0; j < a.top; ++j) {
    // the next in (logit descending, number ascending) order after (last, last_id)
    float best = -INFINITY;
    int id = MP_MAXE;
    for (int e = lane; e < a.experts; e += 32) {
      float v = z[e] + a.bias[e];
      if (!(v == v)) v = -INFINITY;
      const bool after = j == 0 || v < last || (v == last && e > last_id);
      if (after && (v > best || (v == best && e < id))) best = v, id = e;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, id, o);
      if (ov > best || (ov == best && oi < id)) best = ov, id = oi;
    }
    if (j == 0) first = best;
    const float w = first == -INFINITY ? 1.f : expf(best - first);
    sum += w;
    if (lane == 0) a.ids[(size_t)t * slots + j] = min(id, a.experts - 1), a.weight[(size_t)t * slots + j] = w;
    last = best, last_id = id;
  }
  __syncwarp();
  for (int j = lane; j < slots; j += 32) {
    const size_t p = (size_t)t * slots + j;
    if (j >= a.top) a.ids[p] = a.experts + j - a.top, a.weight[p] = 1.f;
    else a.weight[p] /= sum;
  }
}

// The grouped choice.  Identity outputs count as expert number experts + pieces.
__device__ __forceinline__ void choose_grouped(const MoePlanArgs& a, int t) {
  const int lane = threadIdx.x & 31, slots = a.top + a.pieces, per = a.outputs / a.groups;
  const float* z = a.z + (size_t)t * a.ldz;
  float top = -INFINITY, sum = 0.f;
  for (int e = lane; e < a.outputs; e += 32) top = fmaxf(top, z[e]);
  top = warp_max(top);
  for (int e = lane; e < a.outputs; e += 32) sum += expf(z[e] - top);
  sum = warp_sum(sum);
  auto score = [&](int e) { return expf(z[e] - top) / sum; };
  auto choice = [&](int e) {
    const float v = score(e) + a.bias[e];
    return v == v ? v : -INFINITY;
  };
  unsigned kept[2] = {0xffffffffu, 0xffffffffu};
  if (a.keep < a.groups) {
    float best[2] = {-INFINITY, -INFINITY};                      // of groups lane and lane + 32
    for (int g = 0; g < a.groups; ++g) {
      float m = -INFINITY;
      for (int e = g * per + lane; e < (g + 1) * per; e += 32) m = fmaxf(m, choice(e));
      m = warp_max(m);
      if (lane == (g & 31)) {
        if (g < 32) best[0] = m;
        else best[1] = m;
      }
    }
    int ahead[2] = {0, 0};                                       // groups before this lane's
    for (int g = 0; g < a.groups; ++g) {
      const float m0 = __shfl_sync(0xffffffffu, best[0], g & 31), m1 = __shfl_sync(0xffffffffu, best[1], g & 31), m = g < 32 ? m0 : m1;
      ahead[0] += m > best[0] || (m == best[0] && g < lane);
      ahead[1] += m > best[1] || (m == best[1] && g < lane + 32);
    }
    kept[0] = __ballot_sync(0xffffffffu, lane < a.groups && ahead[0] < a.keep);
    kept[1] = __ballot_sync(0xffffffffu, lane + 32 < a.groups && ahead[1] < a.keep);
  }
  float last = INFINITY;
  int last_id = -1;
  for (int j = 0; j < a.top; ++j) {
    // the next in (choice score descending, number ascending) order after (last, last_id)
    float best = -INFINITY;
    int id = MP_MAXE;
    for (int e = lane; e < a.outputs; e += 32) {
      const int g = e / per;
      if (!((g < 32 ? kept[0] >> g : kept[1] >> (g - 32)) & 1u)) continue;
      const float v = choice(e);
      const bool after = j == 0 || v < last || (v == last && e > last_id);
      if (after && (v > best || (v == best && e < id))) best = v, id = e;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, id, o);
      if (ov > best || (ov == best && oi < id)) best = ov, id = oi;
    }
    if (lane == 0) {
      const int e = min(id, a.outputs - 1);
      a.ids[(size_t)t * slots + j] = e < a.experts ? e : a.experts + a.pieces, a.weight[(size_t)t * slots + j] = score(e) * a.scale;
    }
    last = best, last_id = id;
  }
  for (int j = a.top + lane; j < slots; j += 32) {
    const size_t p = (size_t)t * slots + j;
    a.ids[p] = a.experts + j - a.top, a.weight[p] = a.gate_col >= 0 ? sigmoid_x(z[a.gate_col]) : 1.f;
  }
  __syncwarp();
}
__device__ __forceinline__ void choose_any(const MoePlanArgs& a, int t) {
  if (a.outputs) choose_grouped(a, t);
  else choose_experts(a, t);
}

__global__ void __launch_bounds__(256) moe_topk_kernel(const MoePlanArgs a) {
  pdl_launch_dependents(60);
  pdl_wait();
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (t < a.T) choose_any(a, t);
}

__global__ void __launch_bounds__(MP_THREADS) moe_plan_kernel(const MoePlanArgs a, int choose) {
  __shared__ int s_cnt[MP_MAXE], s_off[MP_MAXE], s_item[MP_MAXE], s_warp[2][32];
  pdl_launch_dependents(61);
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, slots = a.top + a.pieces, n = a.experts + a.pieces, P = a.T * slots;
  if (choose)
    for (int t = warp; t < a.T; t += MP_THREADS / 32) choose_any(a, t);
  for (int e = tid; e < MP_MAXE; e += MP_THREADS) s_cnt[e] = e >= a.experts && e < n ? a.T : 0;
  __syncthreads();
  for (int p = tid; p < P; p += MP_THREADS)
    if (p % slots < a.top) atomicAdd(&s_cnt[a.ids[p]], 1);
  __syncthreads();
  // exclusive sums of rows and of tiles over the experts, two a thread
  const int c0 = s_cnt[2 * tid], c1 = s_cnt[2 * tid + 1];
  const int i0 = 2 * tid < n ? (c0 + a.tile - 1) / a.tile : 0, i1 = 2 * tid + 1 < n ? (c1 + a.tile - 1) / a.tile : 0;      // (own rows have none)
  int rows = c0 + c1, items = i0 + i1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int r = __shfl_up_sync(0xffffffffu, rows, o), i = __shfl_up_sync(0xffffffffu, items, o);
    if (lane >= o) rows += r, items += i;
  }
  if (lane == 31) s_warp[0][warp] = rows, s_warp[1][warp] = items;
  __syncthreads();
  int rb = 0, ib = 0;
  for (int w = 0; w < warp; ++w) rb += s_warp[0][w], ib += s_warp[1][w];
  rows += rb - c0 - c1, items += ib - i0 - i1;
  s_off[2 * tid] = rows, s_off[2 * tid + 1] = rows + c0, s_item[2 * tid] = items, s_item[2 * tid + 1] = items + i0;
  if (tid == MP_THREADS - 1) *a.n_items = min(items + i0 + i1, a.max_items);
  __syncthreads();
  for (int e = warp; e < n; e += MP_THREADS / 32) {
    const int first = s_off[e], cnt = s_cnt[e], it = s_item[e], k = (cnt + a.tile - 1) / a.tile;
    for (int i = lane; i < k; i += 32)
      if (it + i < a.max_items) a.items[it + i] = MoeItem{e, first + i * a.tile, min(a.tile, cnt - i * a.tile), 0};
  }
  __syncthreads();
  for (int p = tid; p < P; p += MP_THREADS) {
    const int t = p / slots, j = p % slots, e = a.ids[p];
    const int row = j < a.top ? atomicAdd(&s_off[e], 1) : s_off[e] + t;
    a.place[p] = e < n ? row : -1, a.token[row] = t;             // own rows stand at the list's end, without tiles
  }
}

// The same for a few pairs: a thread a pair, ranks by counting.
constexpr int MQ_MAX = 256;
__global__ void __launch_bounds__(MQ_MAX) moe_plan_small_kernel(const MoePlanArgs a) {
  __shared__ int s_e[MQ_MAX], s_tiles[MQ_MAX];
  pdl_launch_dependents(61);
  pdl_wait();
  const int tid = threadIdx.x, slots = a.top + a.pieces, P = a.T * slots;
  for (int t = tid >> 5; t < a.T; t += blockDim.x >> 5) choose_any(a, t);
  __syncthreads();
  const int e = tid < P ? a.ids[tid] : 0;
  s_e[tid] = e;
  __syncthreads();
  int row = 0, rank = 0, cnt = 0, item = 0, total = 0;          // rows before, rank among the expert's, its rows, tiles before it
  for (int q = 0; q < P; ++q) {
    const int o = s_e[q];
    row += o < e || (o == e && q < tid), rank += o == e && q < tid, cnt += o == e;
  }
  s_tiles[tid] = rank || e == a.experts + a.pieces ? 0 : (cnt + a.tile - 1) / a.tile;        // an expert's tiles count, and are written, at its first pair
  __syncthreads();
  if (tid >= P) return;
  const bool own = e == a.experts + a.pieces;                   // the token's own row: at the list's end, without tiles
  a.place[tid] = own ? -1 : row, a.token[row] = tid / slots;
  if (rank || (own && row)) return;
  for (int q = 0; q < P; ++q) total += s_tiles[q], item += s_e[q] < e ? s_tiles[q] : 0;
  for (int i = 0; !own && i * a.tile < cnt; ++i)
    if (item + i < a.max_items) a.items[item + i] = MoeItem{e, row + i * a.tile, min(a.tile, cnt - i * a.tile), 0};
  if (row == 0) *a.n_items = min(total, a.max_items);
}

// ---- few rows -----------------------------------------------------------------------------------------------
constexpr int MR_THREADS = 256, MR_WARPS = MR_THREADS / 32, MR_U = 4, MR_PAD = 32, MR_ROWS = 8;
constexpr int MR_SLOT = MR_U * 2 * 512;                        // bytes of a ring stage of one warp
constexpr int MR_SMEM = 216 * 1024;

__device__ __forceinline__ void mr_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint4 mr_lds(uint32_t a) {
  uint4 v;
  asm volatile("ld.shared.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "r"(a) : "memory");
  return v;
}

// x: UP, ACT [T, ldx] input rows by token, DOWN [rows, ldx] gated rows by place.  w: [experts, N, K].
// y: UP bf16 [rows, ldy] act(gate) up, ACT the same with act(row) of every weight row, DOWN fp32 [rows, ldy].  A block walks consecutive row tiles of consecutive items.
template <int KIND, int DEPTH>
__global__ void __launch_bounds__(MR_THREADS)
moe_rows_kernel(const bf16* x, int ldx, const bf16* __restrict__ w, void* y, int ldy, const MoeItem* items, const int* n_items, const int* token,
                int N, int K, int KW, int per_item, int act) {
  extern __shared__ __align__(16) unsigned char mr_smem[];
  __shared__ float s_part[2][MR_WARPS * 16 * MR_ROWS];           // one barrier a tile: the sums of a tile are formed under the next one
  bf16* xs = reinterpret_cast<bf16*>(mr_smem + MR_WARPS * DEPTH * MR_SLOT);     // [8][K + MR_PAD]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int RW = MR_WARPS / KW, wr = warp / KW, wk = warp % KW, ldxs = K + MR_PAD;
  const uint32_t ring = (uint32_t)__cvta_generic_to_shared(mr_smem) + warp * DEPTH * MR_SLOT + lane * 16;
  const int steps = K >> 5, per = (steps + KW - 1) / KW, jb = min(steps, wk * per), je = min(steps, jb + per);
  pdl_enter(KIND == MOE_DOWN ? 63 : 62);
  pdl_wait();
  const long total = (long)*n_items * per_item;
  const int first = (int)(total * blockIdx.x / gridDim.x), end = (int)(total * (blockIdx.x + 1) / gridDim.x);
  // fetch cursor: runs DEPTH - 1 blocks of MR_U steps ahead of the products, across row tiles and items
  int f_tile = first, f_j = jb, f_slot = 0, f_item = first / per_item, f_in = first - f_item * per_item;
  const bf16 *f_w = w, *wa = w, *wb = w;
  auto aim = [&]() {                                           // rows of the tile the cursor is on
    const int r0 = (f_in * RW + wr) * 16;
    wa = f_w + (size_t)min(r0 + g, N - 1) * K + (t << 3), wb = f_w + (size_t)min(r0 + g + 8, N - 1) * K + (t << 3);
  };
  if (first < end) f_w = w + (size_t)items[f_item].expert * N * K, aim();
  auto fetch = [&]() {
    if (f_tile < end && jb < je) {
#pragma unroll
      for (int u = 0; u < MR_U; ++u) {
        if (f_j + u < je) {
          const size_t o = (size_t)(f_j + u) << 5;
          cp16(ring + f_slot * MR_SLOT + u * 1024, wa + o);
          cp16(ring + f_slot * MR_SLOT + u * 1024 + 512, wb + o);
        }
      }
      f_j += MR_U;
      if (f_j >= je) {
        f_j = jb, ++f_tile;
        if (++f_in == per_item) {
          f_in = 0, ++f_item;
          if (f_tile < end) f_w = w + (size_t)items[f_item].expert * N * K;
        }
        aim();
      }
    }
    f_slot = f_slot + 1 == DEPTH ? 0 : f_slot + 1;
    cp_commit();
  };
#pragma unroll
  for (int i = 0; i < DEPTH - 1; ++i) fetch();
  int slot = 0, item = first / per_item, in = first - item * per_item, buf = 0;
  bool fresh = true;
  MoeItem it = {0, 0, 0, 0};
  for (int tile = first; tile < end; ++tile, ++in, buf ^= 1) {
    if (in == per_item) in = 0, ++item, fresh = true;
    if (fresh) {
      fresh = false;
      it = items[item];
      __syncthreads();
      for (int m = 0; m < it.n; ++m) {
        const bf16* src = x + (size_t)(KIND != MOE_DOWN ? token[it.row0 + m] : it.row0 + m) * ldx;
        for (int c = threadIdx.x; c < K / 8; c += MR_THREADS)
          *reinterpret_cast<uint4*>(xs + (size_t)m * ldxs + 8 * c) = *reinterpret_cast<const uint4*>(src + 8 * c);
      }
      __syncthreads();
    }
    if (tile + 1 == end) pdl_trigger();
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int j0 = jb; j0 < je; j0 += MR_U) {
      fetch();
      cp_wait<DEPTH - 1>();
      uint4 va[MR_U], vb[MR_U];
#pragma unroll
      for (int u = 0; u < MR_U; ++u) {
        va[u] = mr_lds(ring + slot * MR_SLOT + u * 1024);
        vb[u] = mr_lds(ring + slot * MR_SLOT + u * 1024 + 512);
      }
      slot = slot + 1 == DEPTH ? 0 : slot + 1;
#pragma unroll
      for (int u = 0; u < MR_U; ++u) {
        if (j0 + u < je) {
          uint4 xv = make_uint4(0u, 0u, 0u, 0u);               // rows the tile does not have count as zeros
          if (g < it.n) xv = *reinterpret_cast<const uint4*>(xs + (size_t)g * ldxs + ((j0 + u) << 5) + (t << 3));
          mr_mma(acc, va[u].x, vb[u].x, va[u].y, vb[u].y, xv.x, xv.y);
          mr_mma(acc, va[u].z, vb[u].z, va[u].w, vb[u].w, xv.z, xv.w);
        }
      }
    }
    // accumulator e: weight row g + 8 (e / 2), activation row 2 t + e % 2
#pragma unroll
    for (int e = 0; e < 4; ++e) s_part[buf][(warp * MR_ROWS + 2 * t + (e & 1)) * 16 + g + (e >> 1) * 8] = acc[e];
    __syncthreads();
    auto total_of = [&](int m, int c) {
      float v = 0.f;
      for (int k = 0; k < KW; ++k) v += s_part[buf][(((c >> 4) * KW + k) * MR_ROWS + m) * 16 + (c & 15)];
      return v;
    };
    constexpr int PER = KIND == MOE_UP ? 8 : 16;               // outputs of 16 weight rows
    for (int i = threadIdx.x; i < RW * PER * it.n; i += MR_THREADS) {
      const int m = i / (RW * PER), c = i % (RW * PER) * (16 / PER), n = in * RW * 16 + c;
      if (n >= N) continue;
      const float v = total_of(m, c);
      if (KIND == MOE_UP) reinterpret_cast<bf16*>(y)[(size_t)(it.row0 + m) * ldy + n / 2] = __float2bfloat16(glu_x(v, total_of(m, c + 1), act, 0.f));
      else if (KIND == MOE_ACT) reinterpret_cast<bf16*>(y)[(size_t)(it.row0 + m) * ldy + n] = __float2bfloat16(act_x(v, act));
      else reinterpret_cast<float*>(y)[(size_t)(it.row0 + m) * ldy + n] = v;
    }
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
}

// one warp per output column (UP: pair of weight rows) of an item
template <typename T, int KIND>
__global__ void __launch_bounds__(256)
moe_plain_kernel(const T* x, int ldx, const T* __restrict__ w, void* y, int ldy, const MoeItem* items, const int* n_items, const int* token,
                 int N, int K, int act) {
  constexpr int C = Chunk<T>::N, W = KIND == MOE_UP ? 2 : 1;
  pdl_launch_dependents(64);
  pdl_wait();
  const int lane = threadIdx.x & 31, cols = N / W, ni = *n_items;
  for (long job = blockIdx.x * 8L + (threadIdx.x >> 5); job < (long)ni * cols; job += gridDim.x * 8L) {
    const MoeItem it = items[job / cols];
    const int n = (int)(job % cols);
    const T* wr = w + ((size_t)it.expert * N + (size_t)n * W) * K;
    float acc[MR_ROWS][W];
#pragma unroll
    for (int m = 0; m < MR_ROWS; ++m)
#pragma unroll
      for (int i = 0; i < W; ++i) acc[m][i] = 0.f;
    for (int k = lane * C; k < K; k += 32 * C) {
      float f[W][C];
#pragma unroll
      for (int i = 0; i < W; ++i) Chunk<T>::get(*reinterpret_cast<const uint4*>(wr + (size_t)i * K + k), f[i]);
#pragma unroll
      for (int m = 0; m < MR_ROWS; ++m) {
        if (m < it.n) {
          float v[C];
          Chunk<T>::get(*reinterpret_cast<const uint4*>(x + (size_t)(KIND != MOE_DOWN ? token[it.row0 + m] : it.row0 + m) * ldx + k), v);
#pragma unroll
          for (int i = 0; i < W; ++i)
#pragma unroll
            for (int e = 0; e < C; ++e) acc[m][i] = fmaf(f[i][e], v[e], acc[m][i]);
        }
      }
    }
#pragma unroll
    for (int m = 0; m < MR_ROWS; ++m) {
      if (m < it.n) {
        const float a0 = warp_sum(acc[m][0]), a1 = warp_sum(acc[m][W - 1]);
        if (lane == 0) {
          if (KIND == MOE_UP) reinterpret_cast<T*>(y)[(size_t)(it.row0 + m) * ldy + n] = from_f<T>(glu_x(a0, a1, act, 0.f));
          else if (KIND == MOE_ACT) reinterpret_cast<T*>(y)[(size_t)(it.row0 + m) * ldy + n] = from_f<T>(act_x(a0, act));
          else reinterpret_cast<float*>(y)[(size_t)(it.row0 + m) * ldy + n] = a0;
        }
      }
    }
  }
}

__global__ void __launch_bounds__(256) moe_gather_kernel(const uint4* x, int ld, const int* token, uint4* out, int rows, int chunks) {
  pdl_launch_dependents(65);
  pdl_wait();
  for (int r = blockIdx.x; r < rows; r += gridDim.x) {
    const uint4* src = x + (size_t)token[r] * ld;
    for (int c = threadIdx.x; c < chunks; c += 256) out[(size_t)r * chunks + c] = src[c];
  }
}

int mr_sms() {
  static int n = [] {
    int dev = 0, v = 148;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev);
    return v;
  }();
  return n;
}

template <int KIND, int DEPTH>
cudaError_t rows_launch(const void* x, int ldx, const void* w, void* y, int ldy, const void* items, const void* n_items, const void* token,
                        int groups, int likely, int N, int K, int act, size_t smem, cudaStream_t st) {
  // split K over the warps of a block: shares of at least 16 steps, more splits where a block would get fewer than eight tiles
  // (the blocks' tile counts differ by one)
  int KW = 1;
  while (KW < MR_WARPS && (K / 32 / (2 * KW) >= 16 || (long)groups * likely * KW < 8L * mr_sms() * MR_WARPS)) KW *= 2;
  const int RW = MR_WARPS / KW, per_item = (groups + RW - 1) / RW;
  auto kern = moe_rows_kernel<KIND, DEPTH>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MR_SMEM);
    if (e != cudaSuccess) return e;
    cudaFuncSetAttribute(kern, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    configured = true;
  }
  return trl_launch(kern, dim3(mr_sms()), dim3(MR_THREADS), smem, st, (const bf16*)x, ldx, (const bf16*)w, y, ldy, (const MoeItem*)items,
                    (const int*)n_items, (const int*)token, N, K, KW, per_item, act);
}

}  // namespace

// Experts and places of T tokens (args: filled by the caller).  items: room for max_items >= min(T * slots, experts + pieces) +
// T * slots / tile tiles.
TRL_API int trl_moe_plan(const MoePlanArgs* args, void* stream) {
  const MoePlanArgs& a = *args;
  const int outputs = a.outputs ? a.outputs : a.experts;
  if (a.T <= 0 || a.experts <= 0 || a.top <= 0 || a.top > outputs || a.pieces < 0 || a.experts + a.pieces >= MP_MAXE || outputs > MP_MAXE || a.ldz < outputs ||
      (a.outputs && (a.outputs < a.experts || a.groups < 1 || a.groups > 64 || a.keep < 1 || a.keep > a.groups || a.outputs % a.groups ||
                     a.outputs / a.groups * a.keep < a.top || a.gate_col >= a.ldz)) ||
      a.tile <= 0 || a.max_items <= 0 || !a.z || !a.bias || !a.ids || !a.weight || !a.place || !a.token || !a.items || !a.n_items)
    return (int)cudaErrorInvalidValue;
  const int choose = a.T <= 64;
  cudaStream_t st = (cudaStream_t)stream;
  cudaError_t e = cudaSuccess;
  const int pairs = a.T * (a.top + a.pieces);
  if (pairs <= MQ_MAX && a.T <= 32) return (int)trl_launch(moe_plan_small_kernel, dim3(1), dim3(pairs <= 64 && a.T <= 2 ? 64 : MQ_MAX), 0, st, a);
  if (!choose) e = trl_launch(moe_topk_kernel, dim3((a.T + 7) / 8), dim3(256), 0, st, a);
  if (e == cudaSuccess) e = trl_launch(moe_plan_kernel, dim3(1), dim3(MP_THREADS), 0, st, a, choose);
  return (int)e;
}

// Up (kind 0), down (kind 1) or plain up (kind 2) projections of all tiles (of at most 8 rows each).  likely: a guess of their number.  plain: CUDA cores.
TRL_API int trl_moe_rows(const void* x, int ldx, const void* w, void* y, int ldy, const void* items, const void* n_items, const void* token,
                         int N, int K, int kind, int act, int likely, int f32, void* stream) {
  if (N <= 0 || N % 2 || K < 64 || K % 64 || ldx % 8 || kind < MOE_UP || kind > MOE_ACT || act < GLU_CLAMPED || act > (kind == MOE_ACT ? (int)ACT_GELU_ERF : (int)GLU_GELU) || likely <= 0 || !items ||
      !n_items || !token || ((uintptr_t)x & 15) || ((uintptr_t)w & 15))
    return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  const size_t xb = (size_t)MR_ROWS * (K + MR_PAD) * sizeof(bf16);
  const size_t deep = xb + (size_t)MR_WARPS * 4 * MR_SLOT, flat = xb + (size_t)MR_WARPS * 2 * MR_SLOT;
  const int groups = (N + 15) / 16;
  if (f32 || flat > (size_t)MR_SMEM) {
#define MOE_PLAIN(TT, KK)                                                                                                          \
  return (int)trl_launch(moe_plain_kernel<TT, KK>, dim3(mr_sms() * 4), dim3(256), 0, st, (const TT*)x, ldx, (const TT*)w, y, ldy,   \
                         (const MoeItem*)items, (const int*)n_items, (const int*)token, N, K, act)
    if (f32 && kind == MOE_UP) MOE_PLAIN(float, MOE_UP);
    if (f32 && kind == MOE_ACT) MOE_PLAIN(float, MOE_ACT);
    if (f32) MOE_PLAIN(float, MOE_DOWN);
    if (kind == MOE_UP) MOE_PLAIN(bf16, MOE_UP);
    if (kind == MOE_ACT) MOE_PLAIN(bf16, MOE_ACT);
    MOE_PLAIN(bf16, MOE_DOWN);
#undef MOE_PLAIN
  }
#define MOE_ROWS(KK, DD, SZ) return (int)rows_launch<KK, DD>(x, ldx, w, y, ldy, items, n_items, token, groups, likely, N, K, act, SZ, st)
  if (deep <= (size_t)MR_SMEM) {
    if (kind == MOE_UP) MOE_ROWS(MOE_UP, 4, deep);
    if (kind == MOE_ACT) MOE_ROWS(MOE_ACT, 4, deep);
    MOE_ROWS(MOE_DOWN, 4, deep);
  }
  if (kind == MOE_UP) MOE_ROWS(MOE_UP, 2, flat);
  if (kind == MOE_ACT) MOE_ROWS(MOE_ACT, 2, flat);
  MOE_ROWS(MOE_DOWN, 2, flat);
#undef MOE_ROWS
}

// out[r] = x[token[r]]: rows of `width` 16-bit values, a multiple of 8.
TRL_API int trl_moe_gather(const void* x, int ldx, const void* token, void* out, int rows, int width, void* stream) {
  if (rows <= 0 || width <= 0 || width % 8 || ldx % 8 || ((uintptr_t)x & 15) || ((uintptr_t)out & 15)) return (int)cudaErrorInvalidValue;
  return (int)trl_launch(moe_gather_kernel, dim3(min(rows, mr_sms() * 32)), dim3(256), 0, (cudaStream_t)stream, (const uint4*)x, ldx / 8,
                         (const int*)token, (uint4*)out, rows, width / 8);
}

// Softmax attention of single query rows over the paged cache, bfloat16: grouped heads that are not mixed, keys and values in planes of any two
// widths, with what may stand around the softmax of the general kernel (attention_mixed.cu) as parameters:
//   score_h(j) = (q_h . k_j) * scale, bounded by softcap * tanh(score / softcap) if softcap > 0;  visible: j <= position;
//   out_h = sum_j e^score v_j / (sum_j e^score + e^sink_h)              (sinks optional, one per head)
//   out_h times sigmoid(gate)                                           (gate optional: one number per head, or one per element)
//
// The work is cut as in attention_decode_core.cuh: a CTA per (row, key/value head, part of its keys); a key/value head's query heads are the 16 rows of
// an MMA; every warp walks tiles of 32 keys of its own through a ring of asynchronous copies, keeps its own running maximum, sum and outputs in
// registers (scores and weights never leave them), and no barrier is met before the end, where the warps' results are put
// together in shared memory.  The parts of a row meet in global memory; the CTA that arrives last puts them together.
// Nothing is prefetched before the dependency wait: the keys of this step are written by the kernel before.
//
// Compile-time: KEY_DIM (at most 256), VALUE_DIM (at most 128), both multiples of 16; DECODE_WARPS.
#include "common.cuh"
#include "mma_utils.cuh"

#ifndef KEY_DIM
#define KEY_DIM 64
#endif
#ifndef VALUE_DIM
#define VALUE_DIM 64
#endif

namespace tlie {

constexpr int kD = KEY_DIM, kVD = VALUE_DIM;
constexpr int kKeys = 32;
constexpr int kKRow = kD + 8, kVRow = kVD + 8;                  // padded shared-memory rows (elements)
constexpr int kStages = 2;
constexpr size_t kStageBytes = (size_t)kKeys * (kKRow + kVRow) * sizeof(__nv_bfloat16);
#ifdef DECODE_WARPS
constexpr int kWarps = DECODE_WARPS;
#else
constexpr int kWarps = 8 * kStages * kStageBytes <= 200 * 1024 ? 8 : 4;
#endif
constexpr float kLog2e = 1.4426950408889634f;
constexpr size_t kRingBytes = (size_t)kWarps * kStages * kStageBytes;
constexpr size_t kMergeBytes = (size_t)kWarps * 16 * (kVD + 2) * sizeof(float);
constexpr size_t kSmemBytes = kRingBytes > kMergeBytes ? kRingBytes : kMergeBytes;
static_assert(kD % 16 == 0 && kVD % 16 == 0 && kD <= 256 && kVD <= 128 && kSmemBytes <= 227 * 1024, "widths this kernel takes");
constexpr int kMaxTickets = 16384;   // rows * kv_heads a launch may have

struct HeadsDecodeParams {
  const __nv_bfloat16* rows;
  int row_stride, gate_offset, gate_per_head;
  const __nv_bfloat16* k_pages;
  long long k_page_stride;
  const __nv_bfloat16* v_pages;
  long long v_page_stride;
  const int* positions;
  const int* token_seq;
  const int* block_table;
  int table_stride;
  __nv_bfloat16* out;
  float* partial_o;    // [row, head, part, VALUE_DIM], unnormalised
  float* partial_ml;   // [row, head, part, 2]: maximum in units of log2, sum
  int* tickets;
  int heads, kv_heads, page_size, splits;
  float scale, softcap;
  const float* sinks;
};

// one plane's 32 rows of a tile; rows past the last key are zero (their weights are zero too, and 0 * garbage must stay 0)
template <int WIDTH, int ROW>
__device__ __forceinline__ void load_rows(__nv_bfloat16* smem, const __nv_bfloat16* const (&half)[2], const __nv_bfloat16* pages, int key0, int n_keys, int lane) {
  constexpr int kChunks = WIDTH / 8;
#pragma unroll 4
  for (int idx = lane; idx < kKeys * kChunks; idx += 32) {
    const int row = idx / kChunks, chunk = idx - row * kChunks;
    const bool valid = key0 + row < n_keys;
    cp_async_16(smem + row * ROW + chunk * 8, valid ? (row < 16 ? half[0] : half[1]) + (row & 15) * WIDTH + chunk * 8 : pages, valid);
  }
}

__device__ __forceinline__ void load_tile(const HeadsDecodeParams& p, __nv_bfloat16* stage, const int* table, int tile, int n_keys, int kvh, int lane) {
  const int key0 = tile * kKeys;
  const __nv_bfloat16 *k_half[2], *v_half[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {   // a page holds a multiple of 16 keys, so each half of the tile lies in one page
    const int key = key0 + 16 * h;
    const int index = key / p.page_size, slot = key - index * p.page_size;
    const long long page = key < n_keys ? table[index] : 0;
    k_half[h] = p.k_pages + page * p.k_page_stride + ((size_t)kvh * p.page_size + slot) * kD;
    v_half[h] = p.v_pages + page * p.v_page_stride + ((size_t)kvh * p.page_size + slot) * kVD;
  }
  load_rows<kD, kKRow>(stage, k_half, p.k_pages, key0, n_keys, lane);
  load_rows<kVD, kVRow>(stage + kKeys * kKRow, v_half, p.v_pages, key0, n_keys, lane);
}

__device__ __forceinline__ float gate_of(const HeadsDecodeParams& p, int row, int head, int d) {
  const float z = __bfloat162float(p.rows[(size_t)row * p.row_stride + p.gate_offset + (p.gate_per_head ? head : head * kVD + d)]);
  return 1.0f / (1.0f + expf(-z));
}

__global__ void __launch_bounds__(kWarps * 32) heads_decode_kernel(const HeadsDecodeParams p) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __shared__ int last_arrival;
  const int split = blockIdx.x, kvh = blockIdx.y, row = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, t = lane & 3;
  const int group = p.heads / p.kv_heads;
  grid_launch_dependents();
  grid_dependency_wait();
  const int n_keys = p.positions[row] + 1;
  const int* table = p.block_table + (size_t)p.token_seq[row] * p.table_stride;
  const int tiles = (n_keys + kKeys - 1) / kKeys;
  const int per_split = (tiles + p.splits - 1) / p.splits;
  const int tile_begin = split * per_split, tile_end = min(tiles, tile_begin + per_split);
  __nv_bfloat16* ring = reinterpret_cast<__nv_bfloat16*>(smem_raw + (size_t)warp * kStages * kStageBytes);
  constexpr size_t kStageElements = kStageBytes / sizeof(__nv_bfloat16);

  int next_load = tile_begin + warp;
#pragma unroll
  for (int s = 0; s < kStages - 1; ++s) {
    if (next_load < tile_end) load_tile(p, ring + s * kStageElements, table, next_load, n_keys, kvh, lane);
    cp_async_commit();
    next_load += kWarps;
  }
  // query fragments: MMA rows are the query heads of the group
  unsigned qa[kD / 16][4];
  const __nv_bfloat16* q_base = p.rows + (size_t)row * p.row_stride + (size_t)kvh * group * kD;
#pragma unroll
  for (int ks = 0; ks < kD / 16; ++ks) {
    const int c0 = ks * 16 + 2 * t;
    qa[ks][0] = g < group ? *reinterpret_cast<const unsigned*>(q_base + (size_t)g * kD + c0) : 0u;
    qa[ks][1] = g + 8 < group ? *reinterpret_cast<const unsigned*>(q_base + (size_t)(g + 8) * kD + c0) : 0u;
    qa[ks][2] = g < group ? *reinterpret_cast<const unsigned*>(q_base + (size_t)g * kD + c0 + 8) : 0u;
    qa[ks][3] = g + 8 < group ? *reinterpret_cast<const unsigned*>(q_base + (size_t)(g + 8) * kD + c0 + 8) : 0u;
  }
  float o[kVD / 8][4];
#pragma unroll
  for (int i = 0; i < kVD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
  float row_max[2] = {-INFINITY, -INFINITY}, row_sum[2] = {0.0f, 0.0f};
  const bool upper_rows = group > 8;
  const float sl2 = p.scale * kLog2e;
  const float inverse_cap = p.softcap > 0.0f ? p.scale / p.softcap : 0.0f, cap_log2 = p.softcap * kLog2e;

  int stage = 0;
  for (int tile = tile_begin + warp; tile < tile_end; tile += kWarps) {
    if (next_load < tile_end) load_tile(p, ring + ((stage + kStages - 1) % kStages) * kStageElements, table, next_load, n_keys, kvh, lane);
    cp_async_commit();
    next_load += kWarps;
    cp_async_wait<kStages - 1>();
    __syncwarp();
    const __nv_bfloat16* k_smem = ring + stage * kStageElements;
    const __nv_bfloat16* v_smem = k_smem + kKeys * kKRow;
    float s[kKeys / 8][4];
#pragma unroll
    for (int j = 0; j < kKeys / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.0f;
#pragma unroll
    for (int ks = 0; ks < kD / 16; ++ks) {
#pragma unroll
      for (int jp = 0; jp < kKeys / 16; ++jp) {
        unsigned b[4];
        ldmatrix_x4(b, k_smem + ((jp * 2 + (lane >> 4)) * 8 + (lane & 7)) * kKRow + ks * 16 + ((lane >> 3) & 1) * 8);
        mma_bf16(s[jp * 2], qa[ks], b[0], b[1]);
        mma_bf16(s[jp * 2 + 1], qa[ks], b[2], b[3]);
      }
    }
    // scores in units of log2, the bound, the mask of a row's last tile, the running maximum
    const int key0 = tile * kKeys;
    const bool whole = key0 + kKeys <= n_keys;
    unsigned pa[kKeys / 16][4];
    float rescale[2] = {1.0f, 1.0f};
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (r == 1 && !upper_rows) {
#pragma unroll
        for (int j = 0; j < kKeys / 8; ++j) pa[j >> 1][(j & 1) * 2 + 1] = 0u;
        break;
      }
      float tile_max = -INFINITY;
#pragma unroll
      for (int j = 0; j < kKeys / 8; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float v = s[j][2 * r + e];
          v = p.softcap > 0.0f ? cap_log2 * tanhf(v * inverse_cap) : v * sl2;
          if (!whole && key0 + j * 8 + 2 * t + e >= n_keys) v = -INFINITY;
          s[j][2 * r + e] = v;
          tile_max = fmaxf(tile_max, v);
        }
      tile_max = fmaxf(tile_max, __shfl_xor_sync(0xffffffffu, tile_max, 1));
      tile_max = fmaxf(tile_max, __shfl_xor_sync(0xffffffffu, tile_max, 2));
      const float now = fmaxf(row_max[r], tile_max);   // a tile holds at least one key: finite
      rescale[r] = exp2f(row_max[r] - now);
      row_max[r] = now;
      row_sum[r] *= rescale[r];
#pragma unroll
      for (int j = 0; j < kKeys / 8; ++j) {
        const float p0 = exp2_approx(s[j][2 * r] - now), p1 = exp2_approx(s[j][2 * r + 1] - now);
        row_sum[r] += p0 + p1;
        pa[j >> 1][(j & 1) * 2 + r] = pack_bf16(p0, p1);
      }
    }
    if (__any_sync(0xffffffffu, rescale[0] != 1.0f || rescale[1] != 1.0f)) {
#pragma unroll
      for (int i = 0; i < kVD / 8; ++i) {
        o[i][0] *= rescale[0];
        o[i][1] *= rescale[0];
        o[i][2] *= rescale[1];
        o[i][3] *= rescale[1];
      }
    }
#pragma unroll
    for (int kk = 0; kk < kKeys / 16; ++kk) {
#pragma unroll
      for (int np = 0; np < kVD / 16; ++np) {
        unsigned b[4];
        ldmatrix_x4_trans(b, v_smem + (kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7)) * kVRow + np * 16 + (lane >> 4) * 8);
        mma_bf16(o[np * 2], pa[kk], b[0], b[1]);
        mma_bf16(o[np * 2 + 1], pa[kk], b[2], b[3]);
      }
    }
    __syncwarp();   // the warp is done with this stage before it is loaded again
    stage = (stage + 1) % kStages;
  }
  cp_async_wait<0>();
#pragma unroll
  for (int r = 0; r < 2; ++r) {   // a row's sum lies in the four threads of a quad
    row_sum[r] += __shfl_xor_sync(0xffffffffu, row_sum[r], 1);
    row_sum[r] += __shfl_xor_sync(0xffffffffu, row_sum[r], 2);
  }
  __syncthreads();   // every warp is done with its ring: the warps' results take its place
  float* merge_o = reinterpret_cast<float*>(smem_raw);     // [warp][16][kVD]
  float* merge_ml = merge_o + kWarps * 16 * kVD;           // [warp][16][2]
#pragma unroll
  for (int i = 0; i < kVD / 8; ++i) {
    float* base = merge_o + (size_t)warp * 16 * kVD + i * 8 + 2 * t;
    *reinterpret_cast<float2*>(base + (size_t)g * kVD) = make_float2(o[i][0], o[i][1]);
    *reinterpret_cast<float2*>(base + (size_t)(g + 8) * kVD) = make_float2(o[i][2], o[i][3]);
  }
  if (t == 0) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      merge_ml[(warp * 16 + g + 8 * r) * 2] = row_max[r];
      merge_ml[(warp * 16 + g + 8 * r) * 2 + 1] = row_sum[r];
    }
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < group * kVD; idx += kWarps * 32) {
    const int r = idx / kVD, d = idx - r * kVD;
    const int head = kvh * group + r;
    float top = -INFINITY;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) top = fmaxf(top, merge_ml[(w * 16 + r) * 2]);
    const float sink = p.sinks != nullptr ? p.sinks[head] * kLog2e : -INFINITY;
    if (p.splits == 1) top = fmaxf(top, sink);
    float acc = 0.0f, sum = 0.0f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float mine = merge_ml[(w * 16 + r) * 2];
      const float f = mine == -INFINITY ? 0.0f : exp2f(mine - top);
      acc += f * merge_o[((size_t)w * 16 + r) * kVD + d];
      sum += f * merge_ml[(w * 16 + r) * 2 + 1];
    }
    if (p.splits == 1) {
      float v = acc / (p.sinks != nullptr ? sum + exp2f(sink - top) : sum);
      if (p.gate_offset >= 0) v *= gate_of(p, row, head, d);
      p.out[((size_t)row * p.heads + head) * kVD + d] = __float2bfloat16_rn(v);
    } else {
      const size_t slot = ((size_t)row * p.heads + head) * p.splits + split;
      p.partial_o[slot * kVD + d] = acc;
      if (d == 0) {
        p.partial_ml[slot * 2] = top;      // -inf where this part had no keys
        p.partial_ml[slot * 2 + 1] = sum;
      }
    }
  }
  if (p.splits == 1) return;
  // The CTA of this (row, kv head) that arrives last puts the parts together.  No CTA waits for another.
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) last_arrival = atomicAdd(&p.tickets[row * p.kv_heads + kvh], 1) == p.splits - 1;
  __syncthreads();
  if (!last_arrival) return;
  __threadfence();
  // a warp per query head; lane i holds part i's maximum and sum (at most 32 parts); eight parts' outputs are asked for at a time
  for (int r = warp; r < group; r += kWarps) {
    const int head = kvh * group + r;
    const size_t pair = (size_t)row * p.heads + head;
    constexpr int kPerLane = (kVD + 31) / 32;
    const float part_max = lane < p.splits ? __ldcg(p.partial_ml + (pair * p.splits + lane) * 2) : -INFINITY;
    const float part_sum = lane < p.splits ? __ldcg(p.partial_ml + (pair * p.splits + lane) * 2 + 1) : 0.0f;
    const float sink = p.sinks != nullptr ? p.sinks[head] * kLog2e : -INFINITY;
    const float top = fmaxf(warp_max(part_max), sink);
    const float f = part_max == -INFINITY ? 0.0f : exp2f(part_max - top);
    const float sum = warp_sum(f * part_sum) + (p.sinks != nullptr ? exp2f(sink - top) : 0.0f);
    float acc[kPerLane];
#pragma unroll
    for (int i = 0; i < kPerLane; ++i) acc[i] = 0.0f;
    for (int part0 = 0; part0 < p.splits; part0 += 8) {
      float part[8][kPerLane];
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int i = 0; i < kPerLane; ++i) {
          const int d = lane + 32 * i;
          part[j][i] = (part0 + j < p.splits && d < kVD) ? __ldcg(p.partial_o + (pair * p.splits + part0 + j) * kVD + d) : 0.0f;
        }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float fs = __shfl_sync(0xffffffffu, f, (part0 + j) & 31);
#pragma unroll
        for (int i = 0; i < kPerLane; ++i) acc[i] += fs * part[j][i];   // parts past the last were loaded as zeros
      }
    }
#pragma unroll
    for (int i = 0; i < kPerLane; ++i) {
      const int d = lane + 32 * i;
      if (d >= kVD) continue;
      float v = acc[i] / sum;
      if (p.gate_offset >= 0) v *= gate_of(p, row, head, d);
      p.out[pair * kVD + d] = __float2bfloat16_rn(v);
    }
  }
  if (threadIdx.x == 0) p.tickets[row * p.kv_heads + kvh] = 0;   // ready for the next launch
}

}  // namespace tlie

using namespace tlie;

// Scratch: kMaxTickets counters (zero when first used; every launch leaves them zero), then for splits > 1 the parts.
TLIE_EXPORT long long tlie_heads_decode_scratch_floats(int rows, int heads, int splits) { return kMaxTickets + (splits <= 1 ? 0 : (long long)rows * heads * splits * (kVD + 2)); }

// Row i of ``rows`` starts with its query heads and belongs to the request token_seq[i]; ``gate_offset`` < 0: no gate.  ``sinks`` (32-bit [heads]) may be null.
TLIE_EXPORT int tlie_heads_decode(const void* rows, int row_stride, int gate_offset, int gate_per_head, const void* k_pages, long long k_page_stride, const void* v_pages,
                                  long long v_page_stride, const int* positions, const int* token_seq, const int* block_table, int table_stride, void* out, float* scratch,
                                  int tokens, int heads, int kv_heads, int page_size, float scale, float softcap, const float* sinks, int splits, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (kv_heads <= 0 || heads % kv_heads != 0 || heads / kv_heads > 16 || splits < 1 || splits > 32 || scratch == nullptr || (long long)tokens * kv_heads > kMaxTickets ||
      tokens > 65535 || kv_heads > 65535 || page_size % 16 != 0 || row_stride % 2 != 0)
    return (int)cudaErrorInvalidValue;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(heads_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemBytes);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  HeadsDecodeParams p;
  p.rows = (const __nv_bfloat16*)rows;
  p.row_stride = row_stride;
  p.gate_offset = gate_offset;
  p.gate_per_head = gate_per_head;
  p.k_pages = (const __nv_bfloat16*)k_pages;
  p.k_page_stride = k_page_stride;
  p.v_pages = (const __nv_bfloat16*)v_pages;
  p.v_page_stride = v_page_stride;
  p.positions = positions;
  p.token_seq = token_seq;
  p.block_table = block_table;
  p.table_stride = table_stride;
  p.out = (__nv_bfloat16*)out;
  p.tickets = reinterpret_cast<int*>(scratch);
  p.partial_o = scratch + kMaxTickets;
  p.partial_ml = p.partial_o + (size_t)tokens * heads * splits * kVD;
  p.heads = heads;
  p.kv_heads = kv_heads;
  p.page_size = page_size;
  p.splits = splits;
  p.scale = scale;
  p.softcap = softcap;
  p.sinks = sinks;
  return (int)launch_pdl(heads_decode_kernel, dim3(splits, kv_heads, tokens), dim3(kWarps * 32), kSmemBytes, stream, p);
}

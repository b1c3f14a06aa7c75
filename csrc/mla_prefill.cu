// Prefill of multi-head latent attention on tcgen05, in the expanded form, and the gather of latent rows it starts from.
#include "api.h"
#include "attention_tc.cuh"

namespace {

// Per head, queries and keys of up to 128 + 64 columns (the rotary part's key row is shared by all heads) and values of up
// to 128, keys and values dense rows [sum of kv lengths, heads, ..] that the caller expanded from the gathered latent rows
// with the up-projection GEMMs.  The absorbed form the decode kernel uses would contract over 576 and accumulate 512 columns
// per row at a latent of 512; expanded, a prefill chunk costs a quarter of the FLOPs and O fits tensor memory.  Structure as
// for head dim 128 (two query tiles of 128 rows per CTA whose softmax groups alternate on the tensor core, P in tensor
// memory), with key tiles of 64 so that Q (2 x 48 KB) and two stages of K (24 KB) and V (16 KB) fit shared memory.  The
// rotary block of Q and K comes through tensor maps of its own; an instance without it serves layers without positions.
// Narrower heads are filled with zeros by TMA.  A sliding window drops the key tiles in front of the CTA's first row and
// masks the tiles its lower edge crosses.  The sigmoid of a gate (per element or per head) may multiply the output, and a sink
// per head adds its exponential to the softmax's denominator.
//
// Reference parity: pegainfer-kernels/csrc/k3/k3_flash_mla_prefill.cu (gather / expand, then a dense SM100 FMHA).
constexpr int MV_BYTES = BKV2 * 128 * 2; // 16 KB: [2 blocks of 64 columns][64 rows][128 B]

struct MlaTcParams {
  bf16* out;             // [T, heads * vdim]
  const int* q_indptr;   // [num_seqs + 1]
  const int* kv_indptr;  // [num_seqs + 1] rows of the dense K / V
  const int* kv_lens;    // [num_seqs] keys of a sequence among the dense rows (its last ones)
  int num_seqs, heads, vdim, window;
  int head_major;        // order of the two outer coordinates of the query maps: 1 (row, head), 0 (head, row)
  const bf16* gate;      // [T, heads * vdim] rows of stride ld_gate, or null
  long long ld_gate;
  int gate_cols;         // columns of the gate per head: vdim, or 1 for a gate per (token, head)
  const float* sink;     // [heads], or null
  float scale_log2;
  uint32_t* status;
};

template <bool ROT>
__global__ void __launch_bounds__(THREADS, 1) mla_prefill_tc_kernel(const __grid_constant__ CUtensorMap tm_qn, const __grid_constant__ CUtensorMap tm_qpe,
                                                                    const __grid_constant__ CUtensorMap tm_kn, const __grid_constant__ CUtensorMap tm_kpe,
                                                                    const __grid_constant__ CUtensorMap tm_v, const MlaTcParams p) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = smem_u32(smem_raw);
  uint8_t* tiles = smem_raw + (((base + 1023u) & ~1023u) - base);
  constexpr int QKB = ROT ? 3 : 2;             // 64-column blocks of queries and keys
  constexpr int MQ_BYTES = 128 * QKB * 128;    // [blocks][128 rows][128 B]
  constexpr int MK_BYTES = BKV2 * QKB * 128;   // [blocks][64 rows][128 B]
  uint8_t* q_tile = tiles;                    // GROUPS x 48 KB
  uint8_t* k_tile = tiles + GROUPS * MQ_BYTES;  // 2 x 24 KB
  uint8_t* v_tile = k_tile + 2 * MK_BYTES;    // 2 x 16 KB
  TcSmem* sh = reinterpret_cast<TcSmem*>(v_tile + 2 * MV_BYTES);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = (int)(blockIdx.x % (unsigned)p.heads);
  int b = 0, tile_in_seq = 0;  // late tiles (most keys) first, every head's before any early tile
  {
    int rem = (int)(gridDim.x / (unsigned)p.heads) - 1 - (int)(blockIdx.x / (unsigned)p.heads);
    for (; b < p.num_seqs; ++b) {
      const int n = p.q_indptr[b + 1] - p.q_indptr[b];
      const int nt = (n + BQ2 - 1) / BQ2;
      if (rem < nt) {
        tile_in_seq = rem;
        break;
      }
      rem -= nt;
    }
    if (b >= p.num_seqs) return;
  }
  if (threadIdx.x == 0) {
    mbar_init(&sh->q_full, 1);
    for (int s2 = 0; s2 < 2; ++s2) {
      mbar_init(&sh->k_full[s2], 1);
      mbar_init(&sh->k_empty[s2], 1);
      mbar_init(&sh->v_full[s2], 1);
      mbar_init(&sh->v_empty[s2], 1);
    }
    for (int g = 0; g < GROUPS; ++g) {
      mbar_init(&sh->s_full[g], 1);
      mbar_init(&sh->p_ready[g], 4);
      mbar_init(&sh->o_full[g], 1);
    }
    sh->abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_qn);
    tma_prefetch_desc(&tm_kn);
    if (ROT) {
      tma_prefetch_desc(&tm_qpe);
      tma_prefetch_desc(&tm_kpe);
    }
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 1) {
    tmem_alloc(&sh->tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = sh->tmem_slot;  // columns: S / P of group g at 128 g (64 used), O of group g at 256 + 128 g
  volatile int* abort_flag = &sh->abort_flag;
  PG_PDL_ENTRY();

  const int q0 = p.q_indptr[b], q_len = p.q_indptr[b + 1] - q0;
  const int kv_len = p.kv_lens[b], kv0 = p.kv_indptr[b];
  const int row_base = tile_in_seq * BQ2;
  const int rows_here = min(BQ2, q_len - row_base);
  const int pos_base = kv_len - q_len + row_base;
  // key tiles of group g: j0 .. j0 + n_g - 1 (a sliding window drops the tiles in front of the first row's); the loops count from j0
  const int j0 = p.window > 0 ? max(0, pos_base - p.window + 1) / BKV2 : 0;
  int n_g[GROUPS];
#pragma unroll
  for (int g = 0; g < GROUPS; ++g) {
    const int rows_of_g = min(128, rows_here - g * 128);
    n_g[g] = (rows_of_g > 0 && kv_len > 0) ? min(pos_base + g * 128 + rows_of_g - 1, kv_len - 1) / BKV2 + 1 - j0 : 0;
  }
  const int n_tiles = max(n_g[0], n_g[1]);

  if (warp == 0) {
    if (n_tiles > 0) {
      const uint64_t pol = l2_policy_evict_normal();
      if (lane == 0) {
        mbar_expect_tx(&sh->q_full, GROUPS * MQ_BYTES);
#pragma unroll
        for (int g = 0; g < GROUPS; ++g) {
          const int row = q0 + row_base + g * 128;
          const int y = p.head_major ? row : h, z = p.head_major ? h : row;
          tma_load_3d(q_tile + g * MQ_BYTES, &tm_qn, &sh->q_full, 0, y, z, pol);            // unrotated columns 0 .. 63
          tma_load_3d(q_tile + g * MQ_BYTES + 16384, &tm_qn, &sh->q_full, 64, y, z, pol);   // unrotated columns 64 .. 127
          if (ROT) tma_load_3d(q_tile + g * MQ_BYTES + 32768, &tm_qpe, &sh->q_full, 0, h, row, pol);
        }
      }
      // five boxes per tile, one lane each: K nope (2), K rotary, V (2)
      bool ok = true;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int st = j & 1;
        const int row = kv0 + (j0 + j) * BKV2;  // rows past the sequence belong to the next one (or are filled with zeros): masked
        if (j >= 2) {
          const uint32_t par = (uint32_t)(((j >> 1) - 1) & 1);
          ok = mbar_wait(&sh->k_empty[st], par, abort_flag) && mbar_wait(&sh->v_empty[st], par, abort_flag);
          ok = __all_sync(0xFFFFFFFFu, ok);
          if (!ok) break;
        }
        if (lane == 0) {
          mbar_expect_tx(&sh->k_full[st], MK_BYTES);
          mbar_expect_tx(&sh->v_full[st], MV_BYTES);
        }
        __syncwarp();
        if (lane < 2) tma_load_3d(k_tile + st * MK_BYTES + lane * 8192, &tm_kn, &sh->k_full[st], lane * 64, h, row, pol);
        else if (ROT && lane == 2) tma_load_2d(k_tile + st * MK_BYTES + 16384, &tm_kpe, &sh->k_full[st], 0, row, pol);
        else if (lane == 3 || lane == 4) tma_load_3d(v_tile + st * MV_BYTES + (lane - 3) * 8192, &tm_v, &sh->v_full[st], (lane - 3) * 64, h, row, pol);
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && n_tiles > 0) {
      constexpr uint32_t idesc_s = idesc_bf16(128, BKV2, 0);
      constexpr uint32_t idesc_o = idesc_bf16(128, 128, 1);
      constexpr uint32_t lbo = 8192u, sbo = 1024u;
      bool ok = mbar_wait(&sh->q_full, 0, abort_flag);
      int k_seen = -1, v_seen = -1;
      auto issue_s = [&](int g, int j) {
        if (j >= n_g[g]) return true;
        const int st = j & 1;
        if (k_seen < j) {
          if (!mbar_wait(&sh->k_full[st], (uint32_t)((j >> 1) & 1), abort_flag)) return false;
          k_seen = j;
        }
        tc_fence_after();
        const uint32_t qa = smem_u32(q_tile + g * MQ_BYTES), ka = smem_u32(k_tile + st * MK_BYTES);
#pragma unroll
        for (int cb = 0; cb < QKB; ++cb)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ss(tmem + (uint32_t)(g * 128), umma_desc_k_sw128(qa + cb * 16384 + k * 32), umma_desc_k_sw128(ka + cb * 8192 + k * 32), idesc_s, (cb | k) ? 1u : 0u);
        umma_commit(&sh->s_full[g]);
        const bool last_user = (g == GROUPS - 1) || j >= n_g[GROUPS - 1];
        if (last_user) umma_commit(&sh->k_empty[st]);
        return true;
      };
      auto issue_pv = [&](int g, int j) {
        if (j >= n_g[g]) return true;
        const int st = j & 1;
        if (!mbar_wait(&sh->p_ready[g], (uint32_t)(j & 1), abort_flag)) return false;
        if (v_seen < j) {
          if (!mbar_wait(&sh->v_full[st], (uint32_t)((j >> 1) & 1), abort_flag)) return false;
          v_seen = j;
        }
        tc_fence_after();
        const uint32_t va = smem_u32(v_tile + st * MV_BYTES);
#pragma unroll
        for (int ks = 0; ks < BKV2 / 16; ++ks)
          umma_bf16_ts(tmem + 256u + (uint32_t)(g * 128), tmem + (uint32_t)(g * 128) + (uint32_t)(ks * 8), umma_desc_mn_sw128(va + ks * 2048, lbo, sbo), idesc_o, (j | ks) ? 1u : 0u);
        umma_commit(&sh->o_full[g]);
        const bool last_user = (g == GROUPS - 1) || j >= n_g[GROUPS - 1];
        if (last_user) umma_commit(&sh->v_empty[st]);
        return true;
      };
      ok = ok && issue_s(0, 0) && issue_s(1, 0);
      for (int j = 0; j < n_tiles && ok; ++j) ok = issue_pv(0, j) && issue_s(0, j + 1) && issue_pv(1, j) && issue_s(1, j + 1);
    }
  } else {
    const int g = (warp - 2) >> 2, wq = warp & 3;
    const int r = wq * 32 + lane;
    const int my_n = n_g[g];
    const int pos0 = pos_base + g * 128;
    const int my_pos = pos0 + r;
    const uint32_t s_row = tmem + ((uint32_t)(wq * 32) << 16) + (uint32_t)(g * 128);
    const uint32_t o_row = s_row + 256u;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < my_n && ok; ++j) {
      const int key0 = (j0 + j) * BKV2;
      const bool need_mask = key0 + BKV2 - 1 > min(pos0, kv_len - 1) || (p.window > 0 && key0 <= pos0 + 127 - p.window);
      const int limit = min(my_pos, kv_len - 1) - key0;  // columns lo + 1 .. limit are visible to this row
      const int lo = p.window > 0 ? my_pos - p.window - key0 : -(1 << 30);
      const uint32_t sp = (uint32_t)(j & 1), op = (uint32_t)((j - 1) & 1);
      ok = need_mask ? softmax_tile64<true>(&sh->s_full[g], sp, s_row, o_row, 128, &sh->o_full[g], op, j, limit, lo, p.scale_log2, m, l, &sh->p_ready[g], lane, abort_flag)
                     : softmax_tile64<false>(&sh->s_full[g], sp, s_row, o_row, 128, &sh->o_full[g], op, j, limit, lo, p.scale_log2, m, l, &sh->p_ready[g], lane, abort_flag);
    }
    const int rows_g = min(128, rows_here - g * 128);
    if (ok && my_n > 0) {
      ok = mbar_wait(&sh->o_full[g], (uint32_t)((my_n - 1) & 1), abort_flag);
      tc_fence_after();
    }
    if (p.sink && l > 0.f) l += exp2f(p.sink[h] * 1.4426950408889634f - m);
    float inv = (ok && l > 0.f) ? 1.f / l : 0.f;
    const long long row = q0 + row_base + g * 128 + r;
    if (p.gate && p.gate_cols == 1 && r < rows_g) inv /= 1.f + __expf(-__bfloat162float(p.gate[row * p.ld_gate + h]));
    bf16* dst = p.out + (row * p.heads + h) * p.vdim;
    const bf16* gate = p.gate && p.gate_cols > 1 ? p.gate + row * p.ld_gate + (long long)h * p.vdim : nullptr;
#pragma unroll 1
    for (int c = 0; c < p.vdim; c += 32) {
      uint32_t w[32];
      if (my_n > 0) {  // uniform per group
        tmem_ld32(o_row + c, w);
        tmem_ld_wait();
      }
      if (r < rows_g) {
#pragma unroll
        for (int c8 = 0; c8 < 32; c8 += 8) {
          if (c + c8 >= p.vdim) break;
          float f[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) f[i] = my_n > 0 ? __uint_as_float(w[c8 + i]) * inv : 0.f;
          if (gate) {
            float gv[8];
            unpack8(*reinterpret_cast<const bf16x8*>(gate + c + c8), gv);
#pragma unroll
            for (int i = 0; i < 8; ++i) f[i] /= 1.f + __expf(-gv[i]);
          }
          *reinterpret_cast<bf16x8*>(dst + c + c8) = pack8(f);
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
  if (threadIdx.x == 0 && sh->abort_flag) atomicCAS(p.status, PG_ST_OK, PG_ST_TIMEOUT | (43u << 8));
}

// Latent rows of every key of the step's sequences, through the page table, as dense rows [sum of kv lengths, width];
// `starts`: position of a sequence's first row (null: 0).
__global__ void __launch_bounds__(128) mla_gather_latent_kernel(const bf16* __restrict__ latent, int page_size, long long num_pages, int width, const int* __restrict__ table,
                                                                int table_stride, const int* __restrict__ kv_indptr, const int* __restrict__ starts, int num_seqs, bf16* __restrict__ out, uint32_t* status) {
  PG_PDL_ENTRY();
  const int row = blockIdx.x;
  int b = 0;
  while (b + 1 < num_seqs && kv_indptr[b + 1] <= row) ++b;
  const int pos = row - kv_indptr[b] + (starts ? starts[b] : 0);
  int page = table[(long long)b * table_stride + pos / page_size];
  if (page < 0 || page >= num_pages) {
    if (threadIdx.x == 0) atomicCAS(status, PG_ST_OK, PG_ST_BOUNDS | (44u << 8));
    page = 0;
  }
  const uint4* src = reinterpret_cast<const uint4*>(latent + ((long long)page * page_size + pos % page_size) * width);
  uint4* dst = reinterpret_cast<uint4*>(out + (long long)row * width);
  for (int i = threadIdx.x; i < width / 8; i += blockDim.x) dst[i] = src[i];
}

}  // namespace

// Dense latent rows of the step's keys: latent_layer [pages, page_size, width] -> out [total_kv, width]; `starts` (or null):
// the position of every sequence's first row.
extern "C" int pg_latent_gather(const void* latent_layer, int page_size, long long num_pages, int width, const void* table, int table_stride, const void* kv_indptr, const void* starts, int num_seqs,
                                int total_kv, void* out, void* status, cudaStream_t stream) {
  PG_REQUIRE(width % 8 == 0, "latent width %d is not a multiple of 8", width);
  if (total_kv == 0) return PG_OK;
  PG_CUDA(launch_pdl(mla_gather_latent_kernel, dim3((unsigned)total_kv), dim3(128), 0, stream, (const bf16*)latent_layer, page_size, num_pages, width, (const int*)table,
                     table_stride, (const int*)kv_indptr, (const int*)starts, num_seqs, (bf16*)out, (uint32_t*)status));
  PG_LAUNCH_CHECK();
  return PG_OK;
}

extern "C" int pg_mla_gather_latent(const void* latent_layer, int page_size, long long num_pages, int width, const void* table, int table_stride, const void* kv_indptr,
                                    int num_seqs, int total_kv, void* out, void* status, cudaStream_t stream) {
  return pg_latent_gather(latent_layer, page_size, num_pages, width, table, table_stride, kv_indptr, nullptr, num_seqs, total_kv, out, status, stream);
}

// Expanded-form latent prefill on tcgen05.  q (unrotated columns) and q_pe (rotated ones) by token / head strides, k and v dense
// [total_kv] rows of stride ld_kv with heads dim / vdim columns apart, k_pe rows of stride pe_ld; strides in elements,
// multiples of 8.  kv_lens [num_seqs] counts a sequence's dense rows, which are its last keys; window > 0: a row sees its
// last `window` keys.  out [T, heads * vdim]; gate (or null) rows of stride ld_gate with gate_cols columns per head (vdim, or 1);
// sink f32 [heads] (or null).  `q_tiles` = sum over the sequences of
// ceil(query rows / 256).
extern "C" int pg_latent_prefill_tc(const void* q, long long q_tok, long long q_head, const void* q_pe, long long pe_tok, long long pe_head, const void* k, const void* v, long long ld_kv, const void* k_pe,
                                    long long pe_ld, const void* gate, long long ld_gate, int gate_cols, const void* sink, void* out, const void* q_indptr, const void* kv_indptr, const void* kv_lens, int num_seqs,
                                    int tokens, int total_kv, int heads, int dim, int rot, int vdim, float scale, int window, int q_tiles, void* status, cudaStream_t stream) {
  PG_REQUIRE(dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 && dim >= 8 && vdim >= 8 && dim <= 128 && rot >= 0 && rot <= 64 && vdim <= 128,
             "tcgen05 latent prefill takes up to 128 + 64 query / key and 128 value columns (got %d + %d, %d)", dim, rot, vdim);
  PG_REQUIRE(gate == nullptr || gate_cols == 1 || gate_cols == vdim, "latent prefill: a gate of %d columns per head", gate_cols);
  PG_REQUIRE(gate == nullptr || gate_cols == 1 || (((uintptr_t)gate & 15) == 0 && ld_gate % 8 == 0), "latent prefill: the gate must start and step on 16-byte boundaries");
  if (q_tiles == 0 || tokens == 0 || total_kv == 0) return PG_OK;
  CUtensorMap tm_qn, tm_qpe, tm_kn, tm_kpe, tm_v;
  auto map3 = [](CUtensorMap* m, const void* ptr, int cols, long long d1, long long s1, long long d2, long long s2, int b1, int b2) {
    cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)d1, (cuuint64_t)d2}, st[2] = {(cuuint64_t)s1 * 2, (cuuint64_t)s2 * 2};
    cuuint32_t box[3] = {64, (cuuint32_t)b1, (cuuint32_t)b2};
    return make_tmap_bf16(m, ptr, 3, dims, st, box);
  };
  // outer dimensions in the order of their strides
  const bool head_major = q_head > q_tok;
  PG_REQUIRE(pe_head <= pe_tok, "latent prefill: rotated query columns are token-major");
  int rc = head_major ? map3(&tm_qn, q, dim, tokens, q_tok, heads, q_head, 128, 1) : map3(&tm_qn, q, dim, heads, q_head, tokens, q_tok, 1, 128);
  if (rc == PG_OK) rc = map3(&tm_kn, k, dim, heads, dim, total_kv, ld_kv, 1, BKV2);
  if (rc == PG_OK) rc = map3(&tm_v, v, vdim, heads, vdim, total_kv, ld_kv, 1, BKV2);
  if (rc == PG_OK && rot) {
    rc = map3(&tm_qpe, q_pe, rot, heads, pe_head, tokens, pe_tok, 1, 128);
    cuuint64_t dims[2] = {(cuuint64_t)rot, (cuuint64_t)total_kv}, st[1] = {(cuuint64_t)pe_ld * 2};
    cuuint32_t box[2] = {64, (cuuint32_t)BKV2};
    if (rc == PG_OK) rc = make_tmap_bf16(&tm_kpe, k_pe, 2, dims, st, box);
  }
  if (rc != PG_OK) return rc;
  if (!rot) tm_qpe = tm_qn, tm_kpe = tm_kn;  // not used by the instance without rotated columns
  MlaTcParams p;
  p.out = (bf16*)out;
  p.q_indptr = (const int*)q_indptr;
  p.kv_indptr = (const int*)kv_indptr;
  p.kv_lens = (const int*)kv_lens;
  p.num_seqs = num_seqs;
  p.heads = heads;
  p.vdim = vdim;
  p.window = window;
  p.head_major = head_major;
  p.gate = (const bf16*)gate;
  p.ld_gate = ld_gate;
  p.gate_cols = gate_cols;
  p.sink = (const float*)sink;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.status = (uint32_t*)status;
  auto smem = [](int blocks) { return 1024 + (size_t)blocks * 128 * (GROUPS * 128 + 2 * BKV2) + 2 * (size_t)MV_BYTES + sizeof(TcSmem) + 64; };
  static bool attr_done = false;
  if (!attr_done) {
    PG_CUDA(cudaFuncSetAttribute(mla_prefill_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem(3)));
    PG_CUDA(cudaFuncSetAttribute(mla_prefill_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem(2)));
    attr_done = true;
  }
  PG_CUDA(launch_pdl(rot ? mla_prefill_tc_kernel<true> : mla_prefill_tc_kernel<false>, dim3((unsigned)q_tiles * (unsigned)heads), dim3(THREADS), smem(rot ? 3 : 2), stream, tm_qn, tm_qpe, tm_kn, tm_kpe, tm_v, p));
  PG_LAUNCH_CHECK();
  return PG_OK;
}

// The 128 + 64 / 128 form with head-major unrotated queries [heads, T, 128] (`q_nope_head_stride` elements between heads: the rows
// may be a prefix of a longer step), q_pe [T, heads, 64], k_nope and v [total_kv, heads, 128] and k_pe = column `pe_col` of
// the dense latent rows [total_kv, pe_ld].
extern "C" int pg_mla_prefill_tc(const void* q_nope_hm, long long q_nope_head_stride, const void* q_pe, const void* k_nope, const void* k_pe_rows, int pe_ld, int pe_col, const void* v, void* out,
                                 const void* q_indptr, const void* kv_indptr, const void* kv_lens, int num_seqs, int tokens, int total_kv, int heads, int nope, int rope, int vdim,
                                 float scale, int q_tiles, void* status, cudaStream_t stream) {
  PG_REQUIRE(nope == 128 && rope == 64 && vdim == 128, "tcgen05 MLA prefill is built for 128 + 64 query / key and 128 value columns (got %d + %d, %d)", nope, rope, vdim);
  return pg_latent_prefill_tc(q_nope_hm, 128, q_nope_head_stride, q_pe, (long long)heads * 64, 64, k_nope, v, (long long)heads * 128, (const bf16*)k_pe_rows + pe_col, pe_ld, nullptr, 0, 0, nullptr, out, q_indptr,
                              kv_indptr, kv_lens, num_seqs, tokens, total_kv, heads, nope, rope, vdim, scale, 0, q_tiles, status, stream);
}

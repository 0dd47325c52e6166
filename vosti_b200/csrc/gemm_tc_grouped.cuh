// Products of experts with their own rows on the tensor cores (included by gemm_tc.cu, whose tile
// geometry, barriers and epilogues they use). The rows of X are sorted by expert: expert e owns the
// rows offsets[e] .. offsets[e + 1] - 1, on the device; its weight is `tiles_per_expert` feature tiles of
// the packed weight (every expert's features padded to whole tiles), so the host decides nothing
// from the choice and a step may be replayed from a CUDA graph.
//
//   Y[r, f] = sum_k X[r, k] * W[expert of r][f, k]
//
// grouped_few (a step of at most 128 tokens; an expert then has at most that many rows): features on
// the MMA's M side as in gemm_tc_kernel; grid (feature tile, n-th expert with rows, K split). Only
// experts with rows have CTAs, so only their weights are read.
// grouped_wide (more): rows on the M side as in gemm_tc_wide_kernel, persistent over the tiles
// (expert, 128 rows, 256 features); a tile's rows beyond its expert's are computed and not stored.

// Epilogues: bfloat16, float32, unsummed K splits, or a gated form (the features then are blocks of 16 gate
// features and their 16 up features): those of gemm_tc.cu, and EPI_CLAMPGLU with a limit L and a constant c,
// g sigmoid(c g) (u + 1) of g = min(gate, L) and u = up clamped to [-L, L]. (It is not one of gemm_tc_kernel's:
// one more branch in that kernel's unrolled epilogue cost the other models' decode steps 2 %.)
constexpr int EPI_CLAMPGLU = 6;
struct GluConstants { float limit, sigmoid_scale; };

__host__ __device__ constexpr bool grouped_is_gated(int epilogue) { return is_gated(epilogue) || epilogue == EPI_CLAMPGLU; }
__device__ __forceinline__ float grouped_gate(int epilogue, float g, float u, const GluConstants& glu) {
  if (epilogue == EPI_CLAMPGLU) {
    return clamped_glu(g, u, glu.limit, glu.sigmoid_scale);
  }
  return gate_act(epilogue, g) * u;
}

// The n-th expert that has rows, and its rows [lo, hi); -1 if there are fewer. Every warp of the block alike.
__device__ __forceinline__ int nth_busy_expert(const int* __restrict__ offsets, int experts, int n, int& lo, int& hi) {
  const int lane = threadIdx.x & 31;
  for (int e0 = 0; e0 < experts; e0 += 32) {
    const int e = e0 + lane;
    const int a = e < experts ? offsets[e] : 0, b = e < experts ? offsets[e + 1] : 0;
    unsigned busy = __ballot_sync(0xffffffffu, b > a);
    const int here = __popc(busy);
    if (n < here) {
      for (int i = 0; i < n; ++i) busy &= busy - 1;
      const int at = __ffs(busy) - 1;
      lo = __shfl_sync(0xffffffffu, a, at);
      hi = __shfl_sync(0xffffffffu, b, at);
      return e0 + at;
    }
    n -= here;
  }
  return -1;
}

// KIND of epilogue, known where the code is laid out so that a kernel's unrolled epilogue holds one form:
// 0 bfloat16; 1 float32 or unsummed splits; 2 a gated form of gemm_tc.cu; 3 the clamped form.
__host__ __device__ constexpr int grouped_kind(int epilogue) {
  return epilogue == EPI_BF16 ? 0 : epilogue == EPI_CLAMPGLU ? 3 : is_gated(epilogue) ? 2 : 1;
}

template <int BN, int STAGES, int KIND>
__global__ void __launch_bounds__(THREADS, 1)
gemm_tc_grouped_few_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x,
                           void* __restrict__ out, const int* __restrict__ offsets, int experts, int rows, int features,
                           int tiles_per_expert, int k_blocks, int ld_out, int epilogue, int w_tiles, int x_rows,
                           const GluConstants glu, unsigned* status) {
  constexpr int B_BYTES = BN * BK * 2;
  constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) uint64_t full_bar[STAGES];
  __shared__ __align__(8) uint64_t empty_bar[STAGES];
  __shared__ __align__(8) uint64_t accum_bar;
  __shared__ uint32_t tmem_base_holder;
  __shared__ volatile int abort_flag;

  pdl_wait();                                          // which experts have rows is the kernel before's answer
  int row_lo = 0, row_hi = 0;
  const int expert = nth_busy_expert(offsets, experts, blockIdx.y, row_lo, row_hi);
  row_lo = max(row_lo, 0);
  const int n = min(min(row_hi, rows) - row_lo, BN);    // (the launcher picks BN so that an expert's rows fit)
  if (expert < 0 || n <= 0) return;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int m0 = blockIdx.x * BM;                      // first feature of the expert's tile
  const int splits = gridDim.z, split = blockIdx.z;
  const int kb_begin = (int)((long long)k_blocks * split / splits);
  const int my_blocks = (int)((long long)k_blocks * (split + 1) / splits) - kb_begin;

  if (threadIdx.x == 0) {
    abort_flag = 0;
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(smem_u32(&full_bar[s]), 1);
      mbar_init(smem_u32(&empty_bar[s]), 1);
    }
    mbar_init(smem_u32(&accum_bar), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(smem_u32(&tmem_base_holder), BN);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_holder;
  pdl_launch_dependents();                             // after the tensor memory is ours: a dependent must not take it first

  if (warp == 0) {
    if (lane == 0) {
      const int w_tile = expert * tiles_per_expert + (int)blockIdx.x;
      for (int i = 0; i < my_blocks; ++i) {
        const int s = i % STAGES;
        if (i >= STAGES && !mbar_wait(smem_u32(&empty_bar[s]), ((i / STAGES) - 1) & 1, &abort_flag, status)) break;
        const uint32_t bar = smem_u32(&full_bar[s]);
        mbar_expect_tx(bar, (uint32_t)(A_BYTES + x_rows * BK * 2));
        const uint32_t dst = smem_u32(smem + s * STAGE_BYTES);
        tma_load_2d(dst, &map_w, 0, ((kb_begin + i) * w_tiles + w_tile) * BM, bar);
        tma_load_2d(dst + A_BYTES, &map_x, (kb_begin + i) * BK, row_lo, bar);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = instr_desc(BN);
      bool ok = true;
      for (int i = 0; i < my_blocks && ok; ++i) {
        const int s = i % STAGES;
        ok = mbar_wait(smem_u32(&full_bar[s]), (i / STAGES) & 1, &abort_flag, status);
        if (!ok) break;
        tc_fence_after();
        const uint32_t a_addr = smem_u32(smem + s * STAGE_BYTES);
        const uint64_t da = smem_desc_sw128(a_addr), db = smem_desc_sw128(a_addr + A_BYTES);
#pragma unroll
        for (int k = 0; k < BK / UMMA_K; ++k) umma_bf16(tmem_base, da + 2 * k, db + 2 * k, idesc, (i > 0 || k > 0) ? 1u : 0u);
        umma_commit(smem_u32(&empty_bar[s]));
      }
      if (ok) umma_commit(smem_u32(&accum_bar));
    }
  } else {
    const int quarter = warp & 3;
    const bool ok = my_blocks > 0 ? mbar_wait_warp(smem_u32(&accum_bar), 0, &abort_flag, status) : true;
    tc_fence_after();
    const int feature = m0 + quarter * 32 + lane;
    if (ok) {
#pragma unroll 1
      for (int c0 = 0; c0 < BN; c0 += 32) {
        if (c0 >= n) break;                               // uniform across the warp
        uint32_t r[32];
        if (my_blocks > 0) {
          tmem_load32(tmem_base + ((uint32_t)(quarter * 32) << 16) + (uint32_t)c0, r);
        } else {
#pragma unroll
          for (int j = 0; j < 32; ++j) r[j] = 0u;
        }
        if (KIND >= 2) {
          bf16* y = reinterpret_cast<bf16*>(out);
          const int out_feature = (m0 + quarter * 32) / 2 + (lane & 15);
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            const float mine = __uint_as_float(r[j]);
            const float other = __shfl_xor_sync(0xffffffffu, mine, 16);
            if (lane < 16 && c0 + j < n && out_feature < ld_out)
              y[(int64_t)(row_lo + c0 + j) * ld_out + out_feature] = __float2bfloat16_rn(grouped_gate(KIND == 3 ? EPI_CLAMPGLU : epilogue, mine, other, glu));
          }
        } else if (feature < features) {
          float* y = reinterpret_cast<float*>(out) + (KIND == 1 && epilogue == EPI_PARTIAL ? (int64_t)split * rows * ld_out : 0);
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            if (c0 + j >= n) continue;
            const int64_t at = (int64_t)(row_lo + c0 + j) * ld_out + feature;
            if (KIND == 0) reinterpret_cast<bf16*>(out)[at] = __float2bfloat16_rn(__uint_as_float(r[j]));
            else y[at] = __uint_as_float(r[j]);
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (abort_flag) {
    for (int i = 0; i < 64; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, BN);
  }
}

// Walks the tiles of grouped_wide in order: tile numbers run over experts, inside an expert over its row tiles
// fastest. `seek` must be called with ascending numbers; false: there is no such tile.
struct GroupedTiles {
  const int* offsets;
  int experts, rows, n_tiles;
  int e = 0, first = 0, lo = 0, hi = 0;                // current expert, number of its first tile, its rows
  __device__ __forceinline__ void read() {
    lo = e < experts ? max(offsets[e], 0) : 0;
    hi = e < experts ? min(offsets[e + 1], rows) : 0;
  }
  __device__ __forceinline__ bool seek(int tile, int& expert, int& m0, int& row_end, int& n0) {
    while (e < experts) {
      const int m_tiles = hi > lo ? (hi - lo + BM - 1) / BM : 0;
      if (tile < first + m_tiles * n_tiles) {
        const int inside = tile - first;
        expert = e;
        m0 = lo + (inside % m_tiles) * BM;
        row_end = hi;
        n0 = (inside / m_tiles) * WIDE_BN;
        return true;
      }
      first += m_tiles * n_tiles;
      ++e;
      read();
    }
    return false;
  }
};

__global__ void __launch_bounds__(THREADS, 1)
gemm_tc_grouped_wide_kernel(const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_w,
                            void* __restrict__ out, const int* __restrict__ offsets, int experts, int rows, int features,
                            int tiles_per_expert, int k_blocks, int ld_out, int epilogue, int w_tiles, const GluConstants glu,
                            unsigned* status) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) uint64_t full_bar[WIDE_STAGES];
  __shared__ __align__(8) uint64_t empty_bar[WIDE_STAGES];
  __shared__ __align__(8) uint64_t acc_full[2];
  __shared__ __align__(8) uint64_t acc_empty[2];
  __shared__ uint32_t tmem_base_holder;
  __shared__ volatile int abort_flag;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    abort_flag = 0;
    for (int s = 0; s < WIDE_STAGES; ++s) {
      mbar_init(smem_u32(&full_bar[s]), 1);
      mbar_init(smem_u32(&empty_bar[s]), 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(smem_u32(&acc_full[a]), 1);
      mbar_init(smem_u32(&acc_empty[a]), 4);       // one arrival per epilogue warp
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(smem_u32(&tmem_base_holder), 2 * WIDE_BN);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_holder;

  pdl_launch_dependents();
  pdl_wait();                                      // the offsets and rows are the kernel before's
  GroupedTiles walk{offsets, experts, rows, (features + WIDE_BN - 1) / WIDE_BN};
  walk.read();
  int expert, m0, row_end, n0;
  if (warp == 0) {
    if (lane == 0) {
      uint32_t it = 0;
      bool ok = true;
      for (int tile = blockIdx.x; ok && walk.seek(tile, expert, m0, row_end, n0); tile += gridDim.x) {
        for (int kb = 0; kb < k_blocks; ++kb, ++it) {
          const int s = it % WIDE_STAGES;
          const uint32_t round = it / WIDE_STAGES;
          if (it >= WIDE_STAGES && !mbar_wait(smem_u32(&empty_bar[s]), (round - 1) & 1, &abort_flag, status)) {
            ok = false;
            break;
          }
          const uint32_t bar = smem_u32(&full_bar[s]);
          mbar_expect_tx(bar, WIDE_STAGE_BYTES);
          const uint32_t a_dst = smem_u32(smem + s * WIDE_STAGE_BYTES);
          tma_load_2d(a_dst, &map_x, kb * BK, m0, bar);
          tma_load_2d(a_dst + A_BYTES, &map_w, 0, (kb * w_tiles + expert * tiles_per_expert + n0 / BM) * BM, bar);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = instr_desc(WIDE_BN);
      uint32_t it = 0, local = 0;
      bool ok = true;
      for (int tile = blockIdx.x; ok && walk.seek(tile, expert, m0, row_end, n0); tile += gridDim.x, ++local) {
        const uint32_t as = local & 1, acc_round = local >> 1;
        if (local >= 2) ok = mbar_wait(smem_u32(&acc_empty[as]), (acc_round - 1) & 1, &abort_flag, status);
        if (!ok) break;
        tc_fence_after();
        const uint32_t d_tmem = tmem_base + as * WIDE_BN;
        for (int kb = 0; kb < k_blocks; ++kb, ++it) {
          const int s = it % WIDE_STAGES;
          ok = mbar_wait(smem_u32(&full_bar[s]), (it / WIDE_STAGES) & 1, &abort_flag, status);
          if (!ok) break;
          tc_fence_after();
          const uint32_t a_addr = smem_u32(smem + s * WIDE_STAGE_BYTES);
          const uint64_t da = smem_desc_sw128(a_addr), db = smem_desc_sw128(a_addr + A_BYTES);
#pragma unroll
          for (int k = 0; k < BK / UMMA_K; ++k) umma_bf16(d_tmem, da + 2 * k, db + 2 * k, idesc, (kb > 0 || k > 0) ? 1u : 0u);
          umma_commit(smem_u32(&empty_bar[s]));
        }
        if (ok) umma_commit(smem_u32(&acc_full[as]));
      }
    }
  } else {
    const int quarter = warp & 3;
    uint32_t local = 0;
    for (int tile = blockIdx.x; walk.seek(tile, expert, m0, row_end, n0); tile += gridDim.x, ++local) {
      const uint32_t as = local & 1;
      if (!mbar_wait_warp(smem_u32(&acc_full[as]), (local >> 1) & 1, &abort_flag, status)) break;
      tc_fence_after();
      const int row = m0 + quarter * 32 + lane;
      const bool row_ok = row < row_end;
#pragma unroll 1
      for (int c0 = 0; c0 < WIDE_BN; c0 += 32) {
        const int f0 = n0 + c0;
        if (f0 >= features) break;
        uint32_t r[32];
        tmem_load32(tmem_base + as * WIDE_BN + ((uint32_t)(quarter * 32) << 16) + (uint32_t)c0, r);
        if (!row_ok) continue;
        if (epilogue == EPI_CLAMPGLU) {
          // columns f0 .. f0 + 15 are gate features, f0 + 16 .. f0 + 31 their up features
          uint32_t packed[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            const __nv_bfloat162 v = __floats2bfloat162_rn(
                grouped_gate(EPI_CLAMPGLU, __uint_as_float(r[2 * j]), __uint_as_float(r[16 + 2 * j]), glu),
                grouped_gate(EPI_CLAMPGLU, __uint_as_float(r[2 * j + 1]), __uint_as_float(r[17 + 2 * j]), glu));
            packed[j] = *reinterpret_cast<const uint32_t*>(&v);
          }
          bf16* y = reinterpret_cast<bf16*>(out) + (int64_t)row * ld_out + f0 / 2;
          if ((ld_out & 7) == 0) {
            reinterpret_cast<uint4*>(y)[0] = make_uint4(packed[0], packed[1], packed[2], packed[3]);
            reinterpret_cast<uint4*>(y)[1] = make_uint4(packed[4], packed[5], packed[6], packed[7]);
          } else {
#pragma unroll
            for (int j = 0; j < 8; ++j) reinterpret_cast<uint32_t*>(y)[j] = packed[j];   // ld_out is even
          }
          continue;
        }
        store_token_columns(r, out, row, f0, features, ld_out, epilogue);
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&acc_empty[as]));
    }
  }
  tc_fence_before();
  __syncthreads();
  if (abort_flag) {
    for (int i = 0; i < 64; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 2 * WIDE_BN);
  }
}

// The K splits of a clamped gated product, summed in split order, through the activation.
__global__ void grouped_clamped_reduce_kernel(const float* __restrict__ partial, bf16* __restrict__ out, int splits, int rows,
                                              int features, const GluConstants glu) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t plane = (int64_t)rows * features, n = plane / 2;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t row = i / (features / 2);
    const int f = (int)(i % (features / 2));
    const float* p = partial + row * features + (f / 16) * 32 + f % 16;
    float g = 0.f, u = 0.f;
    for (int s = 0; s < splits; ++s) {
      g += p[s * plane];
      u += p[s * plane + 16];
    }
    out[i] = __float2bfloat16_rn(grouped_gate(EPI_CLAMPGLU, g, u, glu));
  }
}

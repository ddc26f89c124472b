// Blocks of a thread-block cluster that share a row: a sum over all of them through distributed shared memory, and the
// launch of such a kernel.
#pragma once

#include "common.cuh"
#include <cooperative_groups.h>

namespace ccb {

constexpr int kMaxClusterBlocks = 8;   // (the portable size)

// A block may only write into another one's shared memory once that one runs: cluster_arrive() as the kernel starts,
// cluster_sum() waits for it.  Every thread of every block of the cluster calls both once.
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }

// v: the block's own total, the same in all its threads; slots: shared memory of kMaxClusterBlocks floats.  The blocks'
// totals are added in the order of their ranks.
__device__ __forceinline__ float cluster_sum(float v, float* slots) {
  namespace cg = cooperative_groups;
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
  const cg::cluster_group cluster = cg::this_cluster();
  const int n = (int)cluster.num_blocks();
  if ((int)threadIdx.x < n) cluster.map_shared_rank(slots, (int)threadIdx.x)[cluster.block_rank()] = v;
  cluster.sync();
  float total = 0.f;
  for (int i = 0; i < n; ++i) total += slots[i];
  return total;
}

}  // namespace ccb

// ccb_launch_ex for a kernel whose blocks form clusters of `cluster` neighbours along x (grid.x is a multiple of it).
template <typename... KArgs, typename... Args>
static inline void ccb_launch_cluster(bool early, int cluster, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                      cudaStream_t stream, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = (unsigned)cluster;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  if (g_ccb_pdl && (early || g_ccb_pdl > 1)) {
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.numAttrs = 2;
  }
  cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);  // the error is read by ccb_launch_status()
}

// Kernel launch with optional programmatic stream serialization and an optional cluster along x.
#pragma once
#include <cuda_runtime.h>

namespace nfb {

template <typename K, typename... Args>
cudaError_t launch_kernel(K kern, dim3 grid, dim3 block, size_t smem, cudaStream_t stream, bool pdl, int cluster_x,
                          Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (pdl) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n++].val.programmaticStreamSerializationAllowed = 1;
  }
  if (cluster_x > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = cluster_x; attr[n].val.clusterDim.y = 1; attr[n++].val.clusterDim.z = 1;
  }
  cfg.attrs = attr; cfg.numAttrs = n;
  return cudaLaunchKernelEx(&cfg, kern, args...);
}

}  // namespace nfb

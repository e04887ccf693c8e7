// Shared between the translation units of the dense GEMM (dense_gemm.cu dispatches, dense_umma.cu is the tcgen05 kernel).
#pragma once

#include "host_util.h"

namespace q38 {

struct DenseCall {
  const void* x;
  int ldx, m;
  q38_dense_weight w;
  q38_dense_epilogue ep;
  const q38_gemm_workspace* ws;
};
constexpr int kDenseUmmaTiles = 4;  // token tiles of the tcgen05 kernel
int dense_umma_tile(int index);     // 32, 64, 128, 256 tokens
int dense_umma(const DenseCall& c, int tile_index, cudaStream_t stream);

}  // namespace q38

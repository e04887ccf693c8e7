// Shared between the translation units of the dense GEMM (dense_gemm.cu dispatches, dense_umma.cu is the tcgen05 kernel).
#pragma once

#include "host_util.h"

namespace q38 {

struct DenseCall {
  const void* x;
  int ldx, m;
  q38_dense_weight w;
  q38_dense_groups groups;
  q38_dense_epilogue ep;
  const q38_gemm_workspace* ws;
};
struct DenseUmmaChoice {
  int tok, cluster;  // token tile; CTAs that split one tile's k range
};
bool dense_umma_fits(const DenseCall& c);
DenseUmmaChoice dense_umma_choice(int m, int n, int k, int groups);
inline bool dense_glu(int kind) { return kind == Q38_DENSE_GLU_GELU || kind == Q38_DENSE_GLU_SILU; }
int dense_umma(const DenseCall& c, DenseUmmaChoice choice, cudaStream_t stream);

}  // namespace q38

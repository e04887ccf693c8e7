#include "dense_gemm.h"

// Module of the serving subset (`triune_b200._S`): the GEMM family and the heterogeneous-layer kernels, which is what a
// process that only serves such a model needs to have compiled. The full extension registers the same functions.
#include <torch/extension.h>

void register_gemm(pybind11::module& m);
void register_hybrid(pybind11::module& m);

PYBIND11_MODULE(_S, m) {
  register_gemm(m);
  register_hybrid(m);
}

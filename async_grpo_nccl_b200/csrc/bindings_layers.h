#pragma once
#include <torch/extension.h>

void bind_layer_ops(pybind11::module_& m);
void bind_hybrid_ops(pybind11::module_& m);

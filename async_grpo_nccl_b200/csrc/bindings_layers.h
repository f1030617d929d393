#pragma once
#include <torch/extension.h>

void bind_layer_ops(pybind11::module_& m);

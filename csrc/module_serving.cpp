// The serving extension alone: built where only the rollout engine is going to run (a fraction of the full build).
#include <torch/extension.h>

#include "api.h"

PYBIND11_MODULE(_C_serving, m) { register_serving(m); }

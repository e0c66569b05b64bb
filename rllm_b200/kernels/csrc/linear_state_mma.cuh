#pragma once
#include "linear_state.cuh"

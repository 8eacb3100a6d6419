/* absent.h -- a launcher that refuses because its kernel is not in this library. */
#ifndef VXB_ABSENT_H
#define VXB_ABSENT_H

#include "decoder_state.h"
#include "kernels.h"
#include "nn_device.cuh"
#include "vx_b200.h"

#define NOT_HERE(name)                                                                   \
  name " is not part of this library, which serves one kind of decoder; build the "      \
       "whole one (python -m vx_b200.build)"
#define ABSENT(name, ...)                                                                \
  const char *name(__VA_ARGS__) { return NOT_HERE(#name); }

using Stream = cudaStream_t;

#endif /* VXB_ABSENT_H */

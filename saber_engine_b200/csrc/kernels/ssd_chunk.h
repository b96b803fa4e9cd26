// Chunk form of decayed outer products on the tensor cores (ssd_chunk.cu): prompt portions of bf16 models.
#pragma once
#include "ssd.h"

extern "C" size_t saber_ssd_chunk_floats(const saber::SsdParams* p);      // scratch of a step of M rows; 0: sizes it does not take
int saber_ssd_chunk_launches();
int saber_ssd_chunk_launch(const saber::SsdParams* p, cudaStream_t stream);

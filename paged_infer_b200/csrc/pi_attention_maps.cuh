// Shared between the f32 and the bf16 kernels of multi-map attention.
#pragma once

#include "pi_layered.cuh"

struct MapsParams {
  const float* q;
  size_t stride;
  void* out;
  size_t out_stride;
  const void* base;
  int heads, kv_heads, maps, dim, vdim, dp, vp, block_size, window;
  float scale, eps, lambda, out_scale;
  const int32_t *row_seq, *row_pos, *lens, *tables;
  int max_blocks;
  const float* gate;
  size_t gate_stride;
  int gate_per_head;
  const float *slopes, *sinks, *sigmoid_bias;
  int v_in_k;
};

// bf16 pools: true when the tensor-core kernels hold these sizes.
bool pi_maps_attention_tc_usable(const pi_ctx* ctx, const pi_maps_attention& a, const pi_kv_view& kv);
pi_status pi_launch_maps_attention_tc(pi_ctx* ctx, const MapsParams& p, int out_kind, const pi_seq_batch& b);

// Descriptor of grouped-query attention over a paged cache (paged_attention.cu, paged_prefill.cu); plain data, mirrored by
// the Python bindings.
#pragma once
#include <stdint.h>

struct PkPagedAttention {
  // device pointers
  const float* proj;      // [rows, ld]: queries (H x maps x D) at oq, keys (G x maps x D) at ok, values (G x V) at ov
  const double* freq;     // [R / 2] angular frequencies of the rotated leading part of every query and key
  const int* pos;         // [rows] position of every row
  const int* slot;        // [rows] slot of every row
  void* cache;            // [pages, 64, row]: keys (G x maps x dp), then values (G x vp); bf16 or fp32
  const int* table;       // [slots, table_ld] page of every 64 positions
  float* qx;              // [rows, H x maps, D] rotated queries (null: skip)
  void* qf;               // [rows, H x maps, q_ld] bf16 rotated queries, zero padded (null: skip)
  float* part_o;          // [listed rows, nsplit, H x maps, V]
  float* part_ml;         // [listed rows, nsplit, H x maps, 2] (null for the merge: part_o holds finished outputs, nsplit = 1)
  void* out;              // [rows, ldo], head h at h * V
  uint32_t* status;
  const float* q_norm;    // [D] weight of the norm of every query before the rotation (null: none), k_norm: of every key
  const float* k_norm;
  const float* sink;      // [H x maps] score of a key without a value that every query sees (null: none)
  float* v_first;         // [rows, G x V] values of another layer's same tokens (v_mix)
  int ld, oq, ok, ov;
  int H, G, maps, D, V, R;
  int dp, vp, row;        // widths in the cache (multiples of 8) and elements per cached position
  int table_ld, f32;      // f32: cache and out are fp32
  int window, chunk;      // visible positions of query i: all up to i; i - window < j (window > 0); i / chunk == j / chunk (chunk > 0)
  int q_ld, ldo, nsplit;
  int head_norm;          // outputs of a head are divided by their root mean square
  int neighbours;         // rotated pairs are (2i, 2i + 1) instead of (i, i + R / 2)
  int v_mix;              // 1: values are kept in v_first; 2: v <- (1 - mix) v + mix v_first
  int gate;               // column of proj with one gate per head, sigmoid(gate) multiplies the head's output (-1: none)
  int width;              // columns of out that belong to this layer: those behind H x V are set to zero
  float scale, lambda;    // maps == 2: output = first map - lambda x second map
  float post, eps;        // factor on the outputs (behind the head norm); eps of the norms
  float cap, mix;         // cap > 0: scores become cap tanh(score / cap)
};

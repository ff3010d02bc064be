"""The matrix memory of xLSTM as a mixer of the token-major models, with float32 state per sequence in the cache manager
(net-new; beside `LinearAttentionMixer`, whose decay is a constant per head, and the mixers of gated_recurrent.py).

One fused projection [q | k | v | gate | i | f], then

  one token per sequence   pgk_seq_mlstm_step: gates, state, read-out, per-head norm, weight and output gate in one launch
  longer steps             pgk_seq_mlstm_gates (the log gates and their running maximum), pgk_seq_mlstm_chunks (chunk updates, scan,
                           outputs; three launches over all chunks of a segment), with values wider than one block's columns
                           also pgk_seq_linear_finish (per-head norm, weight, output gate)

and the output projection.  State per slot: S [heads, dim, vdim], n [heads, dim], m [heads].
"""
from __future__ import annotations

from ..._lib import api
from ...core.array import GPUArray
from ...core.stream import current_stream_handle as _st
from ..config import MatrixLSTMSpec
from .linear import LinearRows


class MatrixLSTMMixer:
    queries_per_tile = None              # no attention tiles
    WORKSPACE_FLOATS = 1 << 26           # 256 MB of chunk states at most per segment

    def __init__(self, spec: MatrixLSTMSpec, layer: int, proj: LinearRows, o_proj: LinearRows, i_bias: GPUArray, f_bias: GPUArray,
                 norm_weight: GPUArray, eps: float):
        s = spec
        self.spec, self.layer, self.proj, self.o_proj = spec, layer, proj, o_proj
        self.i_bias, self.f_bias, self.norm_weight, self.eps = i_bias, f_bias, norm_weight, float(eps)
        self.qk_cols, self.v_cols, self.proj_cols = s.heads * s.dim, s.heads * s.vdim, s.proj_cols
        if proj.out_features != self.proj_cols or o_proj.in_features != self.v_cols:
            raise ValueError(f"layer {layer}: the products do not match {s}")
        if i_bias.size != s.heads or f_bias.size != s.heads or norm_weight.size != self.v_cols:
            raise ValueError(f"layer {layer}: gate biases or output weight do not match {s}")
        self.chunk_tokens = int(api.seq_mlstm_chunk_tokens())
        self.fused_finish = bool(api.seq_mlstm_fused_finish(s.vdim))

    @property
    def weight_bytes(self) -> int:
        return self.proj.nbytes + self.o_proj.nbytes

    def key_slices(self, ctx) -> int:
        return 1

    def forward(self, ctx, x: GPUArray, out: GPUArray, cache_index: int | None = None, out_scale: int | None = None,
                state=None) -> None:
        """x [T, W] -> out [T, W]; with out_scale (device pointer of [W] floats) out += out_scale * result.  state: this mixer's
        per-slot arrays in the cache manager ([S, n, m])."""
        T, W = ctx.T, self.proj.in_features
        proj, attn = ctx.buf.proj, ctx.buf.attn
        self.proj.forward(x.device_ptr, W, T, proj.device_ptr, self.proj_cols)
        self.attend(ctx, proj.device_ptr, self.proj_cols, attn.device_ptr, self.v_cols, state)
        if out_scale is None:
            self.o_proj.forward(attn.device_ptr, self.v_cols, T, out.device_ptr, self.o_proj.out_features)
        else:
            self.o_proj.forward_seq(attn.device_ptr, self.v_cols, T, out.device_ptr, self.o_proj.out_features, epilogue=4,
                                    col_scale=out_scale)

    def attend(self, ctx, proj_ptr: int, ld: int, attn_ptr: int, ldo: int, state) -> None:
        """Everything between the two matrix products, on a block of columns of rows of stride ld."""
        s, T = self.spec, ctx.T
        if not state or len(state) != 3:
            raise ValueError(f"layer {self.layer}: the matrix-memory mixer needs its three state arrays")
        k_off, v_off = self.qk_cols, 2 * self.qk_cols
        g_off = v_off + self.v_cols
        i_off, f_off = g_off + self.v_cols, g_off + self.v_cols + s.heads
        S, N, M = (a.device_ptr for a in state)
        seqs_ptr, n_seqs = ctx.seqs()
        rows = (proj_ptr, ld, 0, k_off, v_off, g_off, i_off, f_off, self.i_bias.device_ptr, self.f_bias.device_ptr, s.gate_cap,
                float(s.dim) ** -0.5, self.norm_weight.device_ptr, self.eps, attn_ptr, ldo, S, N, M, seqs_ptr, n_seqs)
        if ctx.max_rows == 1:
            api.seq_mlstm_step(*rows, s.heads, s.dim, s.vdim, _st())
            return
        n_chunks = -(-ctx.max_rows // self.chunk_tokens)
        per = n_seqs * s.heads * s.dim * (s.vdim + 1)
        seg = max(1, min(n_chunks, self.WORKSPACE_FLOATS // per))
        n_gates = -(-int(api.seq_mlstm_gate_floats(T, s.heads)) // 4) * 4
        gates = ctx.workspace(n_gates + seg * per).device_ptr
        ws = gates + 4 * n_gates
        api.seq_mlstm_gates(proj_ptr, ld, i_off, f_off, self.i_bias.device_ptr, self.f_bias.device_ptr, s.gate_cap, M, seqs_ptr, n_seqs,
                            T, s.heads, gates, _st())
        for c0 in range(0, n_chunks, seg):
            api.seq_mlstm_chunks(*rows, T, s.heads, s.dim, s.vdim, gates, c0, min(seg, n_chunks - c0), ws, _st())
        if not self.fused_finish:
            api.seq_linear_finish(attn_ptr, ldo, proj_ptr, ld, g_off, self.norm_weight.device_ptr, T, s.heads, s.vdim, 1, 1, self.eps,
                                  1.0, _st())


__all__ = ["MatrixLSTMMixer"]

"""Gated linear attention as a mixer of the token-major models, with float32 state per sequence in the cache manager (net-new; beside
`LinearAttentionMixer`, whose decay is a constant per head, and `GatedLinearMixer`, which has no keys).

The decay is a number per head, token and key channel, sigmoid(W_2 y + b)^(1 / tau), y the inner columns of the fused projection
[q | k | v | gate | y].  Then

  one token per sequence   pgk_seq_gla_step: decays, state, read-out, per-head norm, weight and gate in one launch
  longer steps             pgk_seq_gla_decays (running sums of the log decays), pgk_seq_gla_chunks (chunk updates, scan, outputs; three
                           launches over all chunks of a segment), with values wider than one block's columns also
                           pgk_seq_linear_finish (per-head norm, weight, gate)

and the output projection.  State per slot: S [heads, dim, vdim].
"""
from __future__ import annotations

from ..._lib import api
from ...core.array import GPUArray
from ...core.stream import current_stream_handle as _st
from ..config import GLAMixerSpec
from .linear import LinearRows


class GLAMixer:
    queries_per_tile = None              # no attention tiles
    WORKSPACE_FLOATS = 1 << 26           # 256 MB of chunk states at most per segment

    def __init__(self, spec: GLAMixerSpec, layer: int, proj: LinearRows, o_proj: LinearRows, decay_up: GPUArray, decay_bias: GPUArray,
                 norm_weight: GPUArray, eps: float):
        """decay_up: W_2 transposed, [gate_rank, heads x dim] float32; norm_weight: [heads x vdim], the shared vector repeated per
        head."""
        s = spec
        self.spec, self.layer, self.proj, self.o_proj = spec, layer, proj, o_proj
        self.decay_up, self.decay_bias, self.norm_weight, self.eps = decay_up, decay_bias, norm_weight, float(eps)
        self.qk_cols, self.v_cols, self.proj_cols = s.heads * s.dim, s.heads * s.vdim, s.proj_cols
        if s.gate_rank < 1 or tuple(decay_up.shape) != (s.gate_rank, self.qk_cols) or decay_bias.size != self.qk_cols:
            raise ValueError(f"layer {layer}: the decay matrices do not match {s}")
        if proj.out_features != self.proj_cols or o_proj.in_features != self.v_cols or norm_weight.size != self.v_cols:
            raise ValueError(f"layer {layer}: the products or the output weight do not match {s}")
        self.chunk_tokens = int(api.seq_gla_chunk_tokens(s.dim, s.vdim))
        if self.chunk_tokens < 1:
            raise ValueError(f"layer {layer}: keys of {s.dim} are too large for the chunked form")
        self.fused_finish = bool(api.seq_gla_fused_finish(s.vdim))

    @property
    def weight_bytes(self) -> int:
        return self.proj.nbytes + self.o_proj.nbytes + self.decay_up.nbytes

    def key_slices(self, ctx) -> int:
        return 1

    def forward(self, ctx, x: GPUArray, out: GPUArray, cache_index: int | None = None, out_scale: int | None = None,
                state=None) -> None:
        """x [T, W] -> out [T, W]; with out_scale (device pointer of [W] floats) out += out_scale * result.  state: this mixer's
        per-slot array in the cache manager ([S])."""
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
        if not state:
            raise ValueError(f"layer {self.layer}: gated linear attention needs its state array")
        k_off, v_off = self.qk_cols, 2 * self.qk_cols
        g_off = v_off + self.v_cols
        y_off = g_off + self.v_cols
        S, w2, b2, w = state[0].device_ptr, self.decay_up.device_ptr, self.decay_bias.device_ptr, self.norm_weight.device_ptr
        q_scale, inv_tau = float(s.dim) ** -0.5, 1.0 / s.tau
        seqs_ptr, n_seqs = ctx.seqs()
        if ctx.max_rows == 1:
            api.seq_gla_step(proj_ptr, ld, 0, k_off, v_off, g_off, y_off, s.gate_rank, w2, b2, inv_tau, q_scale, w, self.eps, attn_ptr,
                             ldo, S, seqs_ptr, n_seqs, s.heads, s.dim, s.vdim, _st())
            return
        n_chunks = -(-ctx.max_rows // self.chunk_tokens)
        per = n_seqs * s.heads * s.dim * (s.vdim + 1)
        seg = max(1, min(n_chunks, self.WORKSPACE_FLOATS // per))
        n_sums = -(-T * self.qk_cols // 4) * 4
        sums = ctx.workspace(n_sums + seg * per).device_ptr
        ws = sums + 4 * n_sums
        api.seq_gla_decays(proj_ptr, ld, y_off, s.gate_rank, w2, b2, inv_tau, seqs_ptr, n_seqs, ctx.max_rows, s.heads, s.dim, sums, _st())
        for c0 in range(0, n_chunks, seg):
            api.seq_gla_chunks(proj_ptr, ld, 0, k_off, v_off, g_off, sums, q_scale, w, self.eps, attn_ptr, ldo, S, seqs_ptr, n_seqs,
                               s.heads, s.dim, s.vdim, c0, min(seg, n_chunks - c0), ws, _st())
        if not self.fused_finish:
            api.seq_linear_finish(attn_ptr, ldo, proj_ptr, ld, g_off, w, T, s.heads, s.vdim, 1, 2, self.eps, 1.0, _st())


__all__ = ["GLAMixer"]

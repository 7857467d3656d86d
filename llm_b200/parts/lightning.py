"""Lightning attention: a linear attention whose memory decays by one fixed number per head.

  q = silu(Wq h), k = silu(Wk h) [heads, dim];   v = silu(Wv h) [heads, vdim]
  S_t = d_h S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t          per head, S [dim, vdim] float32, zero at the start
  out = Wo ( rms(o_t) * g_n * sigmoid(Wg h) )               one rms over all heads together, g_n [heads * vdim]

No cache of keys: the request's whole past is the state, kept in its state slot and carried from step to step.  Three forms
of the recurrence, by what a step brings: single tokens (a kernel that reads and writes the state once, straight from the
projection's partial results), prompt portions in bfloat16 (chunks of 64 tokens on the tensor cores, chained through the
state; silu is taken in the projection's epilogue), and token by token for everything else (float32, short portions, sizes
off the grid).  The state and every sum into it are float32.  Sizes, decays, eps and tensor names are parameters.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import ParamInfo, Part, StateNeed, register_part
from .linear import FUSE_PARTIALS, linear, linear_act
from .recurrent import _segments

_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "out": "o", "norm": "norm"}

CHUNKED = True             # False: prompt portions always walk token by token (in segments)
CHUNKED_FROM_TOKENS = 192  # steps of fewer tokens walk token by token


class LightningAttention(Part):
    role = "mixer"

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, decay, eps: float, names=None,
                 prefix: str = "", dtype=None, device=None):
        super().__init__(prefix, dtype, device)
        if min(hidden_size, num_heads, head_dim, value_dim) <= 0:
            raise ValueError("lightning attention: sizes must be positive")
        if head_dim > 256:
            raise ValueError(f"lightning attention: key size {head_dim} exceeds 256, the most the recurrence kernels take")
        decay = [float(d) for d in decay]
        if len(decay) != num_heads:
            raise ValueError(f"lightning attention: {len(decay)} decays for {num_heads} heads")
        self.hidden_size, self.num_heads, self.head_dim, self.value_dim = hidden_size, num_heads, head_dim, value_dim
        self.eps, self.decay_values = float(eps), decay
        self.names = dict(_NAMES, **(names or {}))
        self.qk_size, self.v_size = num_heads * head_dim, num_heads * value_dim
        self.w_in = None          # [q; k; v; gate] stacked: one product per step
        self.w_qkv = self.w_gate = self.w_o = self.gain = self.decay = None

    def parameters(self):
        n = lambda k: self.name(self.names[k])
        W = self.hidden_size
        return {n("q"): ParamInfo((self.qk_size, W)), n("k"): ParamInfo((self.qk_size, W)), n("v"): ParamInfo((self.v_size, W)),
                n("gate"): ParamInfo((self.v_size, W)), n("out"): ParamInfo((W, self.v_size)),
                n("norm"): ParamInfo((self.v_size,), kind="gain", init="ones_normal")}

    def bind(self, tensors):
        n = lambda k: tensors[self.name(self.names[k])]
        self.w_in = torch.cat([n("q"), n("k"), n("v"), n("gate")], dim=0).contiguous()
        cols = 2 * self.qk_size + self.v_size
        self.w_qkv, self.w_gate = self.w_in[:cols], self.w_in[cols:]
        self.gain, self.w_o = n("norm").contiguous(), n("out").contiguous()
        self.decay = torch.tensor(self.decay_values, dtype=torch.float32, device=self.device)

    def cache_need(self):
        return None

    def state_need(self):
        return StateNeed((self.qk_size * self.value_dim,), torch.float32)

    def _chunked(self, x, T: int, ctx):
        """(q|k|v with silu taken, gate) for the chunk-wise form, or None where the step or the sizes do not take it."""
        H, D, V = self.num_heads, self.head_dim, self.value_dim
        cols = 2 * self.qk_size + self.v_size
        if not CHUNKED or ctx.decode_only or T < CHUNKED_FROM_TOKENS or not ops.lightning_chunks_available(self.dtype, D, V, cols, H):
            return None
        qkv = ctx.workspace.get("lightning_qkv", T, cols, self.dtype)
        if not linear_act(x, self.w_qkv, qkv, T, "silu"):
            return None
        return qkv, linear(x, self.w_gate, ctx.workspace.get("lightning_gate", T, self.v_size, self.dtype), T)

    def forward(self, x: torch.Tensor, ctx, view) -> torch.Tensor:
        T, ws = ctx.n_tokens, ctx.workspace
        H, D, V, QK, VS = self.num_heads, self.head_dim, self.value_dim, self.qk_size, self.v_size
        o = ws.get("lightning_o", T, VS, torch.float32)
        chunked = self._chunked(x, T, ctx)
        if chunked is not None:
            qkv, gate = chunked
            cap = ws.max_rows // ops.LIGHTNING_CHUNK + ctx.cu_tokens.numel()          # chunks of any step: the buffer's size
            scratch = ws.flat("lightning_chunks", ops.lightning_chunk_scratch(cap, H, D, V), torch.float32)
            ops.lightning_chunks(o, qkv[:, :QK], qkv[:, QK:2 * QK], qkv[:, 2 * QK:], self.decay, view.state, ctx, H, D, V, scratch)
            gate_col = 0
        else:
            single = ctx.decode_only and ops.lightning_decode_available(D, V, view.state)
            proj = linear(x, self.w_in, ws.get("lightning_in", T, self.w_in.shape[0], self.dtype), T, allow_partial=single and FUSE_PARTIALS)
            if single:
                ops.lightning_decode(o, proj, self.decay, view.state, ctx, H, D, V)
            else:
                seg, seg_state, seg_decay = _segments(ctx, "lightning", QK * V, QK)
                ops.const_scan(o, proj[:, :QK], proj[:, QK:2 * QK], proj[:, 2 * QK:2 * QK + VS], self.decay, view.state, ctx, H, D, V,
                               seg_len=seg, seg_state=seg_state, seg_decay=seg_decay)
            gate, gate_col = proj, 2 * QK + VS
        normed = ws.get("attn_out", T, VS, self.dtype)
        ops.row_rmsnorm_sigmoid(normed, o, self.gain, gate, gate_col, T, self.eps)
        return linear(normed, self.w_o, ws.get("mixer_out", T, self.hidden_size, self.dtype), T, allow_partial=FUSE_PARTIALS)


register_part("mixer", "lightning", LightningAttention)

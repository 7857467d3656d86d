"""Matrix memory with exponential gates (mLSTM).

  q = Wq h * dim^(-1/2), k = Wk h [heads, dim];   v = Wv h [heads, vdim]
  i = cap tanh((Wi h + bi) / cap), f = logsigmoid(cap tanh((Wf h + bf) / cap))        log gates, one per head
  m_t = max(f + m_{t-1}, i);   S_t = exp(f + m_{t-1} - m_t) S_{t-1} + exp(i - m_t) k_t v_t^T,   n_t alike with k_t alone
  o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
  out = Wo ( rms per head(o) * g_n * sigmoid(Wg h) )                                  g_n [heads * vdim]

No cache of keys: the request's whole past is S, n and m, float32 in its state slot, zero at admission and carried from step to
step.  Three forms of the recurrence, by what a step brings (csrc/mlstm.cu): single tokens, straight from the projection's
unsummed partial results; prompt portions in bfloat16 in chunks of 64 tokens on the tensor cores; token by token for everything
else (float32, short portions, sizes off the grid).  The gates' pre-activations are float32 products in every form.  Sizes, cap,
eps and tensor names are parameters.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import ParamInfo, Part, StateNeed, register_part
from .linear import FUSE_PARTIALS, linear

_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "out": "o", "norm": "norm", "i": "i", "f": "f", "i_bias": "i.b", "f_bias": "f.b"}

CHUNKED = True             # False: prompt portions always walk token by token
CHUNKED_FROM_TOKENS = 128  # steps of fewer tokens walk token by token


class MatrixLSTM(Part):
    role = "mixer"

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, value_dim: int, gate_cap: float, eps: float, names=None,
                 prefix: str = "", dtype=None, device=None):
        super().__init__(prefix, dtype, device)
        if min(hidden_size, num_heads, head_dim, value_dim) <= 0 or not gate_cap > 0:
            raise ValueError("mlstm: sizes and the gates' cap must be positive")
        if head_dim > 256:
            raise ValueError(f"mlstm: key size {head_dim} exceeds 256, the most the recurrence kernels take")
        self.hidden_size, self.num_heads, self.head_dim, self.value_dim = int(hidden_size), int(num_heads), int(head_dim), int(value_dim)
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        self.names = dict(_NAMES, **(names or {}))
        self.qk_size, self.v_size = self.num_heads * self.head_dim, self.num_heads * self.value_dim
        self.gate_col = 2 * (self.qk_size + self.v_size)      # [q; k; v; output gate; i; f] stacked: one product for short steps
        self.w_in = self.w_qkvg = self.w_if = self.b_i = self.b_f = self.w_o = self.gain = None

    def parameters(self):
        n, W, H = lambda k: self.name(self.names[k]), self.hidden_size, self.num_heads
        return {n("q"): ParamInfo((self.qk_size, W)), n("k"): ParamInfo((self.qk_size, W)), n("v"): ParamInfo((self.v_size, W)),
                n("gate"): ParamInfo((self.v_size, W)), n("i"): ParamInfo((H, W)), n("f"): ParamInfo((H, W)),
                n("i_bias"): ParamInfo((H,), kind="gain", init="normal"), n("f_bias"): ParamInfo((H,), kind="gain", init="ones_normal"),
                n("norm"): ParamInfo((self.v_size,), kind="gain", init="ones_normal"), n("out"): ParamInfo((W, self.v_size))}

    def bind(self, tensors):
        n = lambda k: tensors[self.name(self.names[k])]
        rows = [n("q"), n("k"), n("v"), n("gate"), n("i"), n("f")]
        used = self.gate_col + 2 * self.num_heads
        rows.append(rows[0].new_zeros(-used % 4, self.hidden_size))      # rows of the product on the 16-byte grid
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_qkvg, self.w_if = self.w_in[:self.gate_col], self.w_in[self.gate_col:used]
        self.b_i, self.b_f, self.gain, self.w_o = n("i_bias").contiguous(), n("f_bias").contiguous(), n("norm").contiguous(), n("out").contiguous()

    def cache_need(self):
        return None

    def state_need(self):
        return StateNeed((ops.mlstm_state(self.num_heads, self.head_dim, self.value_dim)[2],), torch.float32)

    def forward(self, x: torch.Tensor, ctx, view) -> torch.Tensor:
        T, ws = ctx.n_tokens, ctx.workspace
        H, D, V, QK, VS = self.num_heads, self.head_dim, self.value_dim, self.qk_size, self.v_size
        o = ws.get("mlstm_o", T, VS, torch.float32)
        gates = (self.b_i, self.b_f, self.gate_cap, D ** -0.5, view.state, ctx, H, D, V)
        if (CHUNKED and not ctx.decode_only and T >= CHUNKED_FROM_TOKENS
                and ops.mlstm_chunks_available(self.dtype, D, V, self.gate_col, H)):
            proj = linear(x, self.w_qkvg, ws.get("mlstm_qkvg", T, self.gate_col, self.dtype), T)
            z = linear(x, self.w_if, ws.get("mlstm_if", T, 2 * H, torch.float32), T)
            cap = ws.max_rows // ops.MLSTM_CHUNK + ctx.cu_tokens.numel()          # chunks of any step: the buffers' sizes
            scratch = [ws.flat("mlstm_chunk_" + tag, numel, torch.float32)
                       for tag, numel in zip(("S", "n", "m"), ops.mlstm_chunk_scratch(cap, H, D, V))]
            ops.mlstm_chunks(o, proj[:, :QK], proj[:, QK:2 * QK], proj[:, 2 * QK:2 * QK + VS], z, *gates, scratch)
        else:
            single = ctx.decode_only and ops.mlstm_single_available(D, V, view.state)
            proj = linear(x, self.w_in, ws.get("mlstm_in", T, self.w_in.shape[0], torch.float32), T, allow_partial=single and FUSE_PARTIALS)
            ops.mlstm_scan(o, proj, self.gate_col, *gates, single=single)
        normed = ws.get("attn_out", T, VS, self.dtype)
        ops.head_rmsnorm_sigmoid(normed, o, self.gain, proj, 2 * QK + VS, T, H, self.eps)
        return linear(normed, self.w_o, ws.get("mixer_out", T, self.hidden_size, self.dtype), T, allow_partial=FUSE_PARTIALS)


register_part("mixer", "mlstm", MatrixLSTM)

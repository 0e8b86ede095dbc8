"""mLSTM mixer (xLSTM's matrix memory) as a state-slot layer.

x → one projection to q | k | v | output gate, one to the input and forget gate logits (fp32) → soft-capped exponential gates → matrix
memory ``S [key, value]``, normaliser ``n`` and running maximum ``m`` per (sequence, head), all fp32 → per-head RMS norm, weight, sigmoid
output gate → output projection. Heads are split over TP ranks. The recurrence, head norm and gate are ``ops.mlstm``: a recurrent
kernel for short portions and decoding, chunked tensor-core kernels for longer ones."""
from __future__ import annotations

import torch
import torch.nn as nn

from onecat_vllm import ops
from onecat_vllm.config import ModelConfig
from onecat_vllm.layers.linear import MergedColumnParallelLinear, RowParallelLinear
from onecat_vllm.parallel.state import get_state


class MLSTM(nn.Module):
    def __init__(self, cfg: ModelConfig, layer_idx: int, prefix: str):
        super().__init__()
        tp, H = get_state().tp_size, cfg.mlstm_heads
        if H % tp:
            raise ValueError(f"tensor_parallel_size={tp} does not divide the {H} heads of layer {layer_idx}")
        self.H, self.D, self.V = H // tp, cfg.mlstm_key_dim, cfg.mlstm_value_dim
        self.cap, self.eps = cfg.mlstm_gate_cap, cfg.rms_norm_eps
        self.in_proj_qkvg = MergedColumnParallelLinear(cfg.hidden_size, [H * self.D, H * self.D, H * self.V, H * self.V], quant=cfg.quant,
                                                       prefix=prefix + ".in_proj_qkvg", dtype=cfg.dtype)
        self.gate_if = MergedColumnParallelLinear(cfg.hidden_size, [H, H], quant=None, prefix=prefix + ".gate_if", dtype=cfg.dtype,
                                                  out_dtype=torch.float32)
        self.i_bias = nn.Parameter(torch.zeros(self.H, dtype=torch.float32), requires_grad=False)
        self.f_bias = nn.Parameter(torch.zeros(self.H, dtype=torch.float32), requires_grad=False)
        self.norm_weight = nn.Parameter(torch.ones(self.H * self.V, dtype=cfg.dtype), requires_grad=False)
        self.out_proj = RowParallelLinear(H * self.V, cfg.hidden_size, quant=cfg.quant, prefix=prefix + ".out_proj", dtype=cfg.dtype)
        self.layer_idx = layer_idx

    def load_weight(self, pname: str, w: torch.Tensor, shard=None) -> None:
        """Per-head and per-channel parameters, sharded like the heads."""
        st, p = get_state(), getattr(self, pname)
        p.data.copy_(w.reshape(-1).chunk(st.tp_size, 0)[st.tp_rank].to(p.dtype))

    def state_tensors(self):
        return [((self.H, self.D, self.V), torch.float32), ((self.H, self.D), torch.float32), ((self.H,), torch.float32)]

    def forward(self, x: torch.Tensor, md, state) -> torch.Tensor:
        """``state`` = (S fp32 [slots, H, D, V], n fp32 [slots, H, D], m fp32 [slots, H])."""
        if getattr(md, "gdn_record", None) is not None:
            raise ValueError("speculative decoding is not served for mLSTM layers (their states are not recorded per token)")
        y = ops.mlstm(self.in_proj_qkvg(x), self.gate_if(x), self.i_bias, self.f_bias, self.norm_weight, self.eps, self.cap, self.H, self.D, self.V,
                      state, md)
        return self.out_proj(y)

"""Delta rule with one decay per (head, key channel) as a state-slot layer.

x → one projection to q | k | v | low-rank inputs of the decay and of the output gate | step logits → short causal convolution and SiLU on
q | k | v → unit vectors, fp32 recurrence ``S <- g S; S <- S + k (beta (v - S^T k))^T; o = S^T q`` → per-head RMS norm, weight, low-rank sigmoid
gate → output projection. The recurrence is ``ops.channel_delta``: a recurrent kernel for short portions and decoding, chunked tensor-core
kernels for longer ones."""
from __future__ import annotations

import torch
import torch.nn as nn

from onecat_vllm import ops
from onecat_vllm.config import ModelConfig
from onecat_vllm.layers.linear import LinearBase, ReplicatedLinear
from onecat_vllm.parallel.state import get_state


class ChannelDelta(nn.Module):
    def __init__(self, cfg: ModelConfig, layer_idx: int, prefix: str):
        super().__init__()
        if get_state().tp_size > 1:
            raise ValueError("the delta rule with decays per channel is served with tensor_parallel_size=1")
        self.Hk, self.H = cfg.linear_num_key_heads, cfg.linear_num_value_heads
        self.D, self.V = cfg.linear_key_head_dim, cfg.linear_value_head_dim
        self.sizes = [self.Hk * self.D, self.Hk * self.D, self.H * self.V]
        self.C, self.kw, self.eps = sum(self.sizes), cfg.linear_conv_kernel_dim, cfg.rms_norm_eps
        self.ranks = (cfg.linear_decay_rank or self.D, cfg.linear_gate_rank or self.V)
        kw = dict(quant=None, dtype=cfg.dtype)
        self.in_proj_qkvagb = LinearBase(cfg.hidden_size, self.sizes + [*self.ranks, self.H], "replicated", prefix=prefix + ".in_proj_qkvagb", **kw)
        self.a_proj = ReplicatedLinear(self.ranks[0], self.H * self.D, prefix=prefix + ".a_proj", out_dtype=torch.float32, **kw)
        self.g_proj = ReplicatedLinear(self.ranks[1], self.H * self.V, prefix=prefix + ".g_proj", **kw)
        self.conv_weight = nn.Parameter(torch.zeros(self.C, self.kw, dtype=cfg.dtype), requires_grad=False)
        self.A_log = nn.Parameter(torch.zeros(self.H, dtype=torch.float32), requires_grad=False)
        self.dt_bias = nn.Parameter(torch.ones(self.H * self.D, dtype=torch.float32), requires_grad=False)
        self.norm_weight = nn.Parameter(torch.ones(self.V, dtype=cfg.dtype), requires_grad=False)
        self.out_proj = ReplicatedLinear(self.H * self.V, cfg.hidden_size, quant=cfg.quant, prefix=prefix + ".out_proj", dtype=cfg.dtype)
        self.layer_idx = layer_idx

    def load_weight(self, pname: str, w: torch.Tensor, shard=None) -> None:
        """``conv_q`` / ``conv_k`` / ``conv_v``: rows of the one convolution over q | k | v."""
        if pname.startswith("conv_") and pname[-1] in "qkv" and len(pname) == 6:
            i = "qkv".index(pname[-1])
            p = self.conv_weight.data.narrow(0, sum(self.sizes[:i]), self.sizes[i])
        else:
            p = getattr(self, pname).data
        p.copy_(w.reshape(p.shape).to(p.dtype))

    def state_tensors(self):
        return [(ops.conv_state_shape(self.C, self.kw), None), ((self.H, self.D, self.V), torch.float32)]

    def forward(self, x: torch.Tensor, md, state) -> torch.Tensor:
        """``state`` = (convolution inputs [slots, taps - 1, C], S fp32 [slots, H, D, V])."""
        if getattr(md, "gdn_record", None) is not None:
            raise ValueError("speculative decoding is not served for delta-rule layers with decays per channel (their states are not recorded per token)")
        y = self.in_proj_qkvagb(x)
        C, (ra, rg) = self.C, self.ranks
        qkv = ops.causal_conv(y[:, :C], self.conv_weight, None, state[0], md, silu=True)
        a = self.a_proj(y[:, C: C + ra])
        gate = self.g_proj(y[:, C + ra: C + ra + rg])
        o = ops.channel_delta(qkv, a, y[:, C + ra + rg:], self.A_log, self.dt_bias, state[1], md, self.Hk, self.H, self.D, self.V)
        return self.out_proj(ops.gated_norm(o, gate, self.norm_weight, self.eps, self.H, gate_first=False))

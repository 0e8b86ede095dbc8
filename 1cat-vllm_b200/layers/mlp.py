"""Gated feed-forward: merged gate|up column-parallel GEMM with act(gate)·up (SiLU or the tanh form of GELU) applied in its epilogue,
then the row-parallel down projection (reference: models/llama.py ``LlamaMLP``; layers/activation.py ``SiluAndMul``)."""
from __future__ import annotations

import torch.nn as nn

from onecat_vllm.layers.linear import ColumnParallelLinear, MergedColumnParallelLinear, RowParallelLinear


class MLP(nn.Module):
    def __init__(self, hidden: int, inter: int, quant, prefix: str, dtype, parallel: bool = True, fuse_act: bool = True, act: str = "silu",
                 bias: bool = False):
        """``fuse_act=False`` (LoRA-enabled models) keeps gate|up as a plain GEMM so adapter deltas can be added before the activation.
        ``act="gelu_tanh"`` (GeGLU) is fused for dense weights; the packed-weight GEMM's epilogue implements SiLU·mul only."""
        super().__init__()
        # the fused epilogue has no bias input
        fuse_act = fuse_act and not bias and (act == "silu" or act == "gelu_tanh" and (quant is None or quant.method == "none"))
        self.fuse_act, self.act = fuse_act, act
        self.gate_up_proj = MergedColumnParallelLinear(hidden, [inter, inter], bias=bias, quant=quant, prefix=prefix + ".gate_up_proj",
                                                       dtype=dtype, fuse_silu_mul=fuse_act and act == "silu",
                                                       fuse_gelu_mul=fuse_act and act == "gelu_tanh")
        self.down_proj = RowParallelLinear(inter, hidden, bias=bias, quant=quant, prefix=prefix + ".down_proj", dtype=dtype)

    def forward(self, x):
        h = self.gate_up_proj(x)
        if not self.fuse_act:
            from onecat_vllm import ops
            h = ops.silu_and_mul(h) if self.act == "silu" else ops.gelu_tanh_and_mul(h)
        return self.down_proj(h)


class PlainMLP(nn.Module):
    """Feed-forward without a gate: ``down(act(up(x)))`` with ``act`` = squared ReLU (Arcee) or GELU
    (reference: models/arcee.py ``ArceeMLP``; layers/activation.py ``ReLUSquaredActivation``). The tanh form of GELU is part of the up
    projection's epilogue (``fuse_act=False``, for LoRA-enabled models, keeps it apart); the other activations are elementwise
    PyTorch operations between the two GEMMs."""

    def __init__(self, hidden: int, inter: int, quant, prefix: str, dtype, act: str = "relu2", bias: bool = False, fuse_act: bool = True):
        super().__init__()
        self.act = act
        self.fuse_act = fuse_act and act == "gelu_tanh"
        self.up_proj = ColumnParallelLinear(hidden, inter, bias=bias, quant=quant, prefix=prefix + ".up_proj", dtype=dtype,
                                            fuse_gelu_tanh=self.fuse_act)
        self.down_proj = RowParallelLinear(inter, hidden, bias=bias, quant=quant, prefix=prefix + ".down_proj", dtype=dtype)

    def forward(self, x):
        import torch
        import torch.nn.functional as F
        h = self.up_proj(x)
        if self.fuse_act:
            return self.down_proj(h)
        if self.act == "relu2":
            h = torch.square(F.relu(h))
        elif self.act == "gelu_tanh":
            h = F.gelu(h, approximate="tanh")
        elif self.act == "gelu":
            h = F.gelu(h)
        else:
            h = F.silu(h)
        return self.down_proj(h)


class FeedForwardBlock(PlainMLP):
    """An ungated feed-forward that is a block of its own (NemotronH: every block is ``h + mixer(norm(h))`` and the mixer is a
    Mamba-2 layer, an attention layer or this; reference: models/nemotron_h.py ``NemotronHMLPDecoderLayer``). It takes the place of a
    state-slot mixer in the decoder and declares a one-element state, so the runner and the scheduler need no third kind of layer."""

    def __init__(self, cfg, layer_idx: int, prefix: str):
        super().__init__(cfg.hidden_size, cfg.intermediate_size, cfg.quant, prefix, cfg.dtype, act=cfg.hidden_act, bias=cfg.mlp_bias)

    def state_shapes(self):
        return (1, 1), (1, 1, 1)

    def forward(self, x, md=None, state=None):
        return super().forward(x)

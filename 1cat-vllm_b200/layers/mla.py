"""Multi-head Latent Attention (DeepSeek-V2/V3) in absorbed (MQA-over-latent) form
(reference: models/deepseek_v2.py:870-1075; layers/attention/mla_attention.py:322,1297-1330 ``forward_mqa``;
CPU decode csrc/cpu/mla_decode.cpp). The cache stores one ``kv_lora + rope`` wide latent per token; ``W_UK`` is
folded into the query and ``W_UV`` applied to the attention output, so prefill and decode share one kernel."""
from __future__ import annotations

import torch
import torch.nn as nn

from onecat_vllm import ops
from onecat_vllm.config import ModelConfig
from onecat_vllm.layers.common import RMSNorm, get_rope
from onecat_vllm.layers.linear import ColumnParallelLinear, LinearBase, ReplicatedLinear, RowParallelLinear
from onecat_vllm.ops import ref
from onecat_vllm.parallel.state import get_state


class MLAAttention(nn.Module):
    def __init__(self, cfg: ModelConfig, layer_idx: int, prefix: str, device):
        super().__init__()
        tp = get_state().tp_size
        self.H = cfg.num_attention_heads // tp
        self.nope, self.rope_d, self.vd, self.lora = cfg.qk_nope_head_dim, cfg.qk_rope_head_dim, cfg.v_head_dim, cfg.kv_lora_rank
        self.q_lora = cfg.q_lora_rank
        q, dt, Hg = cfg.quant, cfg.dtype, cfg.num_attention_heads
        qk = self.nope + self.rope_d
        self.fused_in, self.gated, self.interleaved = cfg.mla_fused_in, cfg.attn_output_gate, not cfg.mla_rope_half
        self.head_gate = cfg.attn_head_gate   # one gate logit per head, applied inside the attention kernels
        if Hg % tp:
            raise ValueError(f"tensor_parallel_size={tp} does not divide the {Hg} heads of layer {layer_idx}")
        if self.fused_in:
            # query latent (or the queries themselves) | key/value latent and shared key part | output gate, element by element or one
            # logit per head: everything that reads the block's input, in one GEMM
            if self.gated and self.head_gate:
                raise ValueError("latent attention has an elementwise output gate or one per head, not both")
            sizes = [self.q_lora or Hg * qk, self.lora + self.rope_d] + ([Hg * self.vd] if self.gated else [Hg] if self.head_gate else [])
            self.in_proj_dqkvg = LinearBase(cfg.hidden_size, sizes, "column", quant=q, prefix=prefix + ".in_proj_dqkvg", dtype=dt,
                                            segment_tp=[1 if self.q_lora else tp, 1, tp][: len(sizes)])
        elif self.gated or self.head_gate:
            raise ValueError("the output gate of latent attention is part of the fused input projection")
        if self.q_lora:
            if not self.fused_in:
                self.q_a_proj = ReplicatedLinear(cfg.hidden_size, self.q_lora, quant=q, prefix=prefix + ".q_a_proj", dtype=dt)
            self.q_a_layernorm = RMSNorm(self.q_lora, cfg.rms_norm_eps, dtype=dt)
            self.q_b_proj = ColumnParallelLinear(self.q_lora, Hg * qk, quant=q, prefix=prefix + ".q_b_proj", dtype=dt)
        elif not self.fused_in:
            self.q_proj = ColumnParallelLinear(cfg.hidden_size, Hg * qk, quant=q, prefix=prefix + ".q_proj", dtype=dt)
        if not self.fused_in:
            self.kv_a_proj_with_mqa = ReplicatedLinear(cfg.hidden_size, self.lora + self.rope_d, quant=q, prefix=prefix + ".kv_a_proj_with_mqa", dtype=dt)
        self.kv_a_layernorm = RMSNorm(self.lora, cfg.rms_norm_eps, dtype=dt)
        self.kv_b_proj = ColumnParallelLinear(self.lora, Hg * (self.nope + self.vd), quant=q, prefix=prefix + ".kv_b_proj", dtype=dt)
        self.o_proj = RowParallelLinear(Hg * self.vd, cfg.hidden_size, quant=q, prefix=prefix + ".o_proj", dtype=dt)
        self.rope = get_rope(self.rope_d, cfg.max_model_len, cfg.rope_theta, device, cfg.rope_scaling)
        self.scale = cfg.attn_scale if cfg.attn_scale is not None else qk ** -0.5
        sc = cfg.rope_scaling or {}
        if cfg.attn_scale is None and (sc.get("rope_type") or sc.get("type")) in ("yarn", "deepseek_yarn") and sc.get("mscale_all_dim"):
            # DeepSeek yarn: the softmax scale carries mscale(factor, mscale_all_dim)^2 (reference: models/deepseek_v2.py:483-487)
            from onecat_vllm.ops.ref import yarn_mscale
            m = yarn_mscale(float(sc.get("factor", 1.0)), float(sc["mscale_all_dim"]))
            self.scale *= m * m
        # fp32 residual streams come with fp32 softmax weights: the tensor-core kernels then carry them as two bf16 terms
        self.fine_weights = cfg.residual_fp32
        self.lora_pad, self.rope_pad = self.lora, self.rope_d
        self.prefill_sizes = False   # the expanded prefill kernel has a variant for this layer
        if torch.device(device).type == "cuda" and dt == torch.bfloat16:
            from onecat_vllm.ops import cuda as K
            self.lora_pad, self.rope_pad = K.mla_padded_sizes(self.lora, self.rope_d)
            self.prefill_sizes = self.scale > 0 and self.lora_pad % 8 == 0 and self.rope_pad % 8 == 0
        self.cache_width = self.lora_pad + self.rope_pad   # elements of a cached token: latent | shared key part, each padded for the kernel
        self.sinks = nn.Parameter(torch.zeros(self.H, dtype=torch.float32), requires_grad=False) if cfg.attn_sinks else None
        self._wuk = self._wuv = self._wkv = None

    def load_weight(self, pname: str, w: torch.Tensor, shard=None) -> None:
        """Key and value up-projections stored apart (``uk`` / ``uv``, rows head by head) take their places in ``kv_b_proj``; the sink logits
        are sharded with the heads."""
        st = get_state()
        if pname == "sinks":
            self.sinks.data.copy_(w.narrow(0, st.tp_rank * self.H, self.H))
            return
        n = {"uk": self.nope, "uv": self.vd}[pname]
        o = 0 if pname == "uk" else self.nope
        w = w.view(-1, n, self.lora)[st.tp_rank * self.H: (st.tp_rank + 1) * self.H]
        self.kv_b_proj.weight.data.view(self.H, self.nope + self.vd, self.lora)[:, o:o + n].copy_(w)

    def process_weights_after_loading(self):
        """Runs before the child layers' own repacking (parents come first in ``modules()``): the absorbed ``W_UK`` / ``W_UV`` are
        taken from ``kv_b_proj`` while its checkpoint tensors still exist — a quantised ``kv_b_proj`` is packed for the GEMM
        afterwards and can no longer be dequantised on the host side."""
        self._wuk = self._wuv = self._wkv = None
        self._absorb(self.kv_b_proj.compute_dtype)

    def _absorb(self, dtype):
        if self._wuk is None:
            w = self.kv_b_proj.method.dequantized_weight(self.kv_b_proj).to(dtype).view(self.H, self.nope + self.vd, self.lora)
            w = torch.nn.functional.pad(w, (0, self.lora_pad - self.lora))   # zero columns: the padded latent is zero there as well
            self._wuk = w[:, : self.nope, :].contiguous()  # [H, nope, lora]
            self._wuv = w[:, self.nope:, :].contiguous()  # [H, v, lora]
        return self._wuk, self._wuv

    def forward(self, x, md, latent_cache):
        T, gate, q = x.shape[0], None, None
        if self.fused_in:
            y = self.in_proj_dqkvg(x)
            a = self.q_lora or self.H * (self.nope + self.rope_d)
            n = a + self.lora + self.rope_d
            qa, kv = y[:, :a], y[:, a: n]
            gate = y[:, n:] if self.gated or self.head_gate else None
            if not self.q_lora:
                q, qa = qa, None
        else:
            qa, kv = self.q_a_proj(x) if self.q_lora else None, self.kv_a_proj_with_mqa(x)
        # one kernel: both latent norms, the rotation of the shared key part and the cache insert (no data-dependent shape: the step can
        # be captured in a CUDA graph; padding tokens have no slot)
        qa = ops.mla_prepare(qa, kv, self.q_a_layernorm if self.q_lora else None, self.kv_a_layernorm, md.positions, self.rope.cos_sin, latent_cache,
                             md.slot_mapping, self.lora, self.lora_pad, self.interleaved)
        if q is None:
            q = self.q_b_proj(qa) if self.q_lora else self.q_proj(x)
        o = self._attend(q.view(T, self.H, self.nope + self.rope_d), md, latent_cache, gate if self.head_gate else None).reshape(T, self.H * self.vd)
        return self.o_proj(ops.sigmoid_mul(o, gate) if self.gated else o)

    def _expand(self, lat: torch.Tensor) -> torch.Tensor:
        """Latents ``[rows, lora_pad]`` -> keys and values head by head, both padded to 64 columns."""
        if self.nope % 64 == 0 and self.vd % 64 == 0 and self.lora_pad == self.lora:
            return self.kv_b_proj(lat)
        from onecat_vllm.ops import cuda as K
        if self._wkv is None:
            wuk, wuv = self._absorb(lat.dtype)
            pad = lambda w: torch.nn.functional.pad(w, (0, 0, 0, -w.shape[1] % 64))
            self._wkv = torch.cat([pad(wuk), pad(wuv)], 1).reshape(-1, self.lora_pad).contiguous()
        return K.gemm_bf16(lat, self._wkv)

    def _attend(self, q, md, latent_cache, gate=None):
        """Attention over the cached latents. Single tokens and short portions: the key up-projection is moved to the query and the value one
        to the result. Longer portions on the GPU (bf16): keys and values of the context are expanded and attended to per head."""
        wuk, wuv = self._absorb(q.dtype)
        if q.is_cuda:
            from onecat_vllm.ops import cuda as K
            plan = K.mla_prefill_plan(md, self.H, self.nope, self.rope_d, self.vd, self.lora_pad, q.device) if self.prefill_sizes else None
            o = None
            if plan is None or plan[-1]:
                q_abs = K.per_head_matmul(q[..., : self.nope], wuk)
                o_lat = K.mla_decode(q_abs, q[..., self.nope:], latent_cache, md, self.scale, self.lora_pad, self.rope.cos_sin, self.interleaved,
                                     self.fine_weights, 0 if plan is None else K.MLA_PREFILL_MIN_LEN, self.sinks, gate)
                o = K.per_head_matmul(o_lat, wuv.transpose(1, 2))
            if plan is not None:
                if o is None:
                    o = torch.empty(q.shape[0], self.H, self.vd, dtype=q.dtype, device=q.device)
                K.mla_prefill(plan, q, latent_cache, md, self._expand, o, self.nope, self.rope_d, self.lora_pad, self.scale, self.rope.cos_sin,
                              self.interleaved, self.fine_weights, self.sinks, gate)
            return o
        q_abs = torch.einsum("thn,hnl->thl", q[..., : self.nope], wuk)
        q_pe = ref.rope_rows(q[..., self.nope:], md.positions, self.rope.cos_sin, self.interleaved)
        o_lat = ref.mla_decode(q_abs, q_pe, latent_cache, md.block_table, md.query_start_loc, md.seq_lens, self.scale, self.lora, self.sinks, gate)
        return torch.einsum("thl,hvl->thv", o_lat, wuv)

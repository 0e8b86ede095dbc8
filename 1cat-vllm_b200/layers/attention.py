"""Self-attention block: fused QKV GEMM → (per-head norm) → RoPE + paged-KV insert → paged flash attention
→ (sigmoid output gate) → o_proj (reference: models/llama.py attention; models/qwen3_next.py:505-626 for the
gated variant with per-head q/k RMSNorm and partial rotary).

Further options, each on its own: values that are the keys (one cached tensor), a learned distance bias, first tokens that stay visible
outside the sliding window, one output gate per head applied inside the attention kernel."""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn

from onecat_vllm import ops
from onecat_vllm.config import ModelConfig
from onecat_vllm.layers.common import get_rope
from onecat_vllm.layers.linear import QKGParallelLinear, QKVParallelLinear, RowParallelLinear
from onecat_vllm.ops import ref
from onecat_vllm.parallel.state import get_state


class Attention(nn.Module):
    def __init__(self, cfg: ModelConfig, layer_idx: int, prefix: str, device, qkv_in: Optional[int] = None):
        super().__init__()
        tp = get_state().tp_size
        self.D = cfg.head_dim
        self.gated = cfg.attn_output_gate
        self.kv_shared, self.head_gate = cfg.attn_kv_shared, cfg.attn_head_gate
        if (self.kv_shared or self.head_gate) and (cfg.num_attention_heads % tp or (cfg.num_key_value_heads % tp and tp % cfg.num_key_value_heads)):
            raise ValueError(f"tensor_parallel_size={tp} does not divide the heads of layer {layer_idx}")
        # qkv_in: width of the projection's input when it is not the hidden size (EAGLE-3 feeds [embedding ; hidden])
        if self.kv_shared:
            if self.gated or cfg.qk_norm or cfg.qk_norm_full or layer_idx not in cfg.nope_layers:
                raise ValueError("attention whose values are its keys is served without rotary embedding, q / k norms and the elementwise gate")
            self.qkg_proj = QKGParallelLinear(qkv_in or cfg.hidden_size, cfg.head_dim, cfg.num_attention_heads, cfg.num_key_value_heads,
                                              head_gate=self.head_gate, bias=cfg.attention_bias, quant=cfg.quant, prefix=prefix + ".qkg_proj",
                                              dtype=cfg.dtype)
            self.Hq, self.Hkv = self.qkg_proj.num_heads, self.qkg_proj.num_kv_heads
        else:
            if self.head_gate:
                raise ValueError("the per-head output gate is served for attention whose values are its keys")
            self.qkv_proj = QKVParallelLinear(qkv_in or cfg.hidden_size, cfg.head_dim, cfg.num_attention_heads, cfg.num_key_value_heads,
                                              q_mult=2 if self.gated else 1, bias=cfg.attention_bias, quant=cfg.quant,
                                              prefix=prefix + ".qkv_proj", dtype=cfg.dtype)
            self.Hq, self.Hkv = self.qkv_proj.num_heads, self.qkv_proj.num_kv_heads
        self.window_keep, self.chunk = cfg.attn_window_keep, cfg.attn_chunk
        self.rel_max, self.bias_table = cfg.attn_rel_max, None
        self.rel_bias = nn.Parameter(torch.zeros(cfg.attn_rel_buckets, self.Hq, dtype=torch.float32), requires_grad=False) \
            if cfg.attn_rel_buckets else None
        self.o_proj = RowParallelLinear(cfg.num_attention_heads * cfg.head_dim, cfg.hidden_size, bias=cfg.attn_o_bias, quant=cfg.quant,
                                        prefix=prefix + ".o_proj", dtype=cfg.dtype)
        self.sinks = nn.Parameter(torch.zeros(self.Hq, dtype=torch.float32), requires_grad=False) if cfg.attn_sinks else None
        self._tp_rank = get_state().tp_rank
        self.qk_norm, self.gemma, self.eps = cfg.qk_norm, cfg.gemma_norm, cfg.rms_norm_eps
        if cfg.qk_norm:
            init = torch.zeros if cfg.gemma_norm else torch.ones
            self.q_norm = nn.Parameter(init(cfg.head_dim, dtype=cfg.dtype), requires_grad=False)
            self.k_norm = nn.Parameter(init(cfg.head_dim, dtype=cfg.dtype), requires_grad=False)
        self.rotary_dim = 0 if layer_idx in cfg.nope_layers else cfg.rotary_dim
        self.qk_norm_full = cfg.qk_norm_full
        self.norm_after_rope = cfg.qk_norm and cfg.qk_norm_after_rope
        self.mrope_section = getattr(cfg, "mrope_section", None)  # (temporal, height, width) frequency counts; positions are then [3, T]
        if cfg.qk_norm_full:
            if tp > 1:
                raise ValueError("q / k normalisation over the whole projection is served with tensor_parallel_size=1 only")
            self.q_norm = nn.Parameter(torch.ones(cfg.num_attention_heads * cfg.head_dim, dtype=cfg.dtype), requires_grad=False)
            self.k_norm = nn.Parameter(torch.ones(cfg.num_key_value_heads * cfg.head_dim, dtype=cfg.dtype), requires_grad=False)
        # sliding-window layers may rotate with their own base and without the context-extension rule (Gemma3)
        self.window, self.softcap = cfg.layer_window(layer_idx), cfg.attn_softcap
        local = bool(self.window) and cfg.rope_local_theta is not None
        self.rope = get_rope(self.rotary_dim, cfg.max_model_len, cfg.rope_local_theta if local else cfg.rope_theta, device,
                             None if local else cfg.rope_scaling)
        self.scale = cfg.attn_scale if cfg.attn_scale is not None else cfg.head_dim ** -0.5
        self.layer_idx = layer_idx
        self.qkv_clip = cfg.qkv_clip

    def load_weight(self, pname: str, w: torch.Tensor, shard_id=None) -> None:
        """Parameters that belong to the block itself: the per-head sink logits and the columns of the distance-bias table are sharded
        with the query heads. The table takes as many rows (distance buckets) as the checkpoint has."""
        p = getattr(self, pname)
        if pname == "sinks":
            w = w.narrow(0, self._tp_rank * self.Hq, self.Hq)
        if pname == "rel_bias":
            w = w.narrow(1, self._tp_rank * self.Hq, self.Hq)
            p.data = torch.empty(w.shape, dtype=p.dtype, device=p.device)
        p.data.copy_(w.reshape(p.shape))

    def process_weights_after_loading(self) -> None:
        if self.rel_bias is not None:
            idx = torch.tensor(ref.distance_buckets(self.rel_bias.shape[0], self.rel_max), device=self.rel_bias.device)
            self.bias_table = self.rel_bias.data[idx].t().contiguous()   # [Hq, rel_max + 1]: the bias by distance, last entry for all beyond
        if self.kv_shared and self.qkg_proj.compute_dtype == torch.bfloat16 and self.o_proj.weight.is_cuda:
            self._pad_heads()

    def _pad_heads(self) -> None:
        """The bf16 attention kernels exist for head sizes 64, 128 and 256: other sizes run as the next larger one, with zero rows in the
        projections and zero columns in the output projection (scores and outputs stay the same numbers)."""
        D, pad = self.D, next((d for d in (64, 128, 256) if d >= self.D), None)
        if pad is None:
            raise ValueError(f"head size {D} is not supported (at most 256)")
        if pad == D:
            return
        Hq, Hkv, proj = self.Hq, self.Hkv, self.qkg_proj
        w = proj.weight.data
        q, k, g = w[: Hq * D], w[Hq * D: (Hq + Hkv) * D], w[(Hq + Hkv) * D:]
        rows = lambda t: torch.nn.functional.pad(t.view(-1, D, t.shape[1]), (0, 0, 0, pad - D)).reshape(-1, t.shape[1])
        proj.weight.data = torch.cat([rows(q), rows(k), g]).contiguous()
        o = self.o_proj.weight.data
        self.o_proj.weight.data = torch.nn.functional.pad(o.view(o.shape[0], Hq, D), (0, pad - D)).reshape(o.shape[0], -1).contiguous()
        self.D = pad

    def _forward_shared(self, x: torch.Tensor, md, kv_cache: torch.Tensor) -> torch.Tensor:
        T, D, Hq, Hkv = x.shape[0], self.D, self.Hq, self.Hkv
        qkg = self.qkg_proj(x)
        q = qkg[:, : Hq * D].view(T, Hq, D)
        k = qkg[:, Hq * D: (Hq + Hkv) * D].view(T, Hkv, D)
        ops.kv_insert(k, kv_cache, md.slot_mapping)
        o = ops.paged_attention(q, kv_cache, md, self.scale, window=self.window, softcap=self.softcap, sinks=self.sinks, keep=self.window_keep,
                                bias_table=self.bias_table, chunk=self.chunk, gate=qkg[:, (Hq + Hkv) * D:] if self.head_gate else None)
        return self.o_proj(o.reshape(T, Hq * D))

    def forward(self, x: torch.Tensor, md, kv_cache: torch.Tensor) -> torch.Tensor:
        if self.kv_shared:
            return self._forward_shared(x, md, kv_cache)
        T = x.shape[0]
        D, Hq, Hkv = self.D, self.Hq, self.Hkv
        qkv = self.qkv_proj(x)
        if self.qkv_clip is not None:      # OLMo: projections clamped to ±clip before the rotary embedding
            qkv = qkv.clamp(-self.qkv_clip, self.qkv_clip)
        qw = Hq * D * (2 if self.gated else 1)
        if self.gated:
            qg = qkv[:, :qw].view(T, Hq, 2 * D)
            q, gate = qg[..., :D], qg[..., D:]
        else:
            q, gate = qkv[:, :qw].view(T, Hq, D), None
        k = qkv[:, qw:qw + Hkv * D].view(T, Hkv, D)
        v = qkv[:, qw + Hkv * D:].view(T, Hkv, D)
        if self.qk_norm_full:
            q = ops.rms_norm(q.reshape(T, Hq * D), self.q_norm, self.eps)[0].view(T, Hq, D)
            k = ops.rms_norm(k.reshape(T, Hkv * D), self.k_norm, self.eps)[0].view(T, Hkv, D)
        if self.norm_after_rope:
            # rotate first (no cache write), normalise per head, then insert the normalised keys with a zero-width rotation
            q, k = q.contiguous(), k.contiguous()
            ops.rope_and_cache(q, k, v, md.positions, self.rope.cos_sin, None, md.slot_mapping, self.rotary_dim, None, None, self.eps, False)
            q = ops.rms_norm(q.view(T * Hq, D), self.q_norm, self.eps, None, self.gemma)[0].view(T, Hq, D)
            k = ops.rms_norm(k.view(T * Hkv, D), self.k_norm, self.eps, None, self.gemma)[0].view(T, Hkv, D)
            ops.rope_and_cache(q, k, v, md.positions, self.rope.cos_sin[:, :0], kv_cache, md.slot_mapping, 0, None, None, self.eps, False)
        else:
            mrope = self.mrope_section if md.mrope_positions is not None else None
            ops.rope_and_cache(q, k, v, md.mrope_positions if mrope else md.positions, self.rope.cos_sin, kv_cache, md.slot_mapping, self.rotary_dim,
                               self.q_norm if self.qk_norm else None, self.k_norm if self.qk_norm else None, self.eps, self.gemma,
                               mrope_section=mrope)
        o = ops.paged_attention(q, kv_cache, md, self.scale, window=self.window, softcap=self.softcap, sinks=self.sinks, keep=self.window_keep,
                                bias_table=self.bias_table, chunk=self.chunk)
        if gate is not None:
            o = o * torch.sigmoid(gate.float()).to(o.dtype)
        return self.o_proj(o.reshape(T, Hq * D))


class TalkingAttention(nn.Module):
    """Attention whose values are its unnormalised keys and whose heads' softmax weights are mixed by a learned matrix before they meet the values
    (talking heads). Queries and keys are normalised over the whole projection, queries take a temperature that grows with the position, and
    ``r1 ln(1 + r2 distance)`` is taken off the scores.

    One cached row per token serves as key and value: the key norm's weight moves into the queries, its factor is one number per token that is
    cached beside the pages and multiplies the scores. fused q|k GEMM -> norm, temperature and cache insert (one kernel) -> attention in one walk
    over the keys (the mix is linear: every head keeps its weighted sums over the rows of all key heads, and the normalised sums are mixed
    afterwards) -> output projection."""

    kv_shared, token_scale, window, window_keep, bias_table = True, True, 0, 0, None   # what the runner and the graphs ask of an attention layer

    def __init__(self, cfg: ModelConfig, layer_idx: int, prefix: str, device):
        super().__init__()
        if get_state().tp_size > 1:
            raise ValueError("talking-heads attention (norms over the whole projection, weights mixed over all heads) is served with tensor_parallel_size=1")
        if not (cfg.attn_kv_shared and cfg.qk_norm_full and cfg.attn_log_bias) or cfg.attn_softcap or cfg.attn_sinks or cfg.layer_window(layer_idx) or \
                cfg.attn_chunk:
            raise ValueError("talking-heads attention is served with shared keys and values, norms over the whole projection and the logarithmic "
                             "distance bias, over the whole context")
        self.Hq, self.Hkv, self.dim = cfg.num_attention_heads, cfg.num_key_value_heads, cfg.head_dim
        self.qkg_proj = QKGParallelLinear(cfg.hidden_size, self.dim, self.Hq, self.Hkv, bias=cfg.attention_bias, quant=cfg.quant,
                                          prefix=prefix + ".qkg_proj", dtype=cfg.dtype)
        self.o_proj = RowParallelLinear(self.Hq * self.dim, cfg.hidden_size, bias=cfg.attn_o_bias, quant=cfg.quant, prefix=prefix + ".o_proj",
                                        dtype=cfg.dtype)
        ones = lambda n, dt: nn.Parameter(torch.ones(n, dtype=dt), requires_grad=False)
        self.q_norm, self.k_norm = ones(self.Hq * self.dim, cfg.dtype), ones(self.Hkv * self.dim, cfg.dtype)
        self.r1, self.r2 = ones(self.Hq, torch.float32), ones(self.Hq, torch.float32)
        self.talk = nn.Parameter(torch.eye(self.Hq, dtype=cfg.dtype), requires_grad=False)
        self.register_buffer("q_gain", torch.ones(self.Hq * self.dim, dtype=torch.float32), persistent=False)
        self.register_buffer("bias", torch.zeros(2, self.Hq, dtype=torch.float32), persistent=False)
        self.scale = cfg.attn_scale if cfg.attn_scale is not None else self.dim ** -0.5
        self.temperature, self.eps = cfg.attn_temperature, cfg.rms_norm_eps
        tc = torch.device(device).type == "cuda" and cfg.dtype == torch.bfloat16
        self.D = ops.ext().talk_row(self.Hq, self.Hkv, self.dim) if tc else self.dim   # width of a cached row
        self.layer_idx = layer_idx

    def load_weight(self, pname: str, w: torch.Tensor, shard_id=None) -> None:
        getattr(self, pname).data.copy_(w)

    def process_weights_after_loading(self) -> None:
        k = self.k_norm.data.float().view(self.Hkv, 1, self.dim).expand(-1, self.Hq // self.Hkv, -1).reshape(-1)
        self.q_gain.copy_(self.q_norm.data.float() * k * self.scale)
        self.bias.copy_(torch.stack([self.r1.data, self.r2.data]))

    def forward(self, x: torch.Tensor, md, kv_cache) -> torch.Tensor:
        pages, k_scale = kv_cache
        q = ops.talk_prepare(self.qkg_proj(x), self.q_gain, self.eps, self.temperature, md.positions, pages, k_scale, md.slot_mapping, self.Hq, self.Hkv,
                             self.dim)
        o = ops.talk_attention(q, pages, k_scale, md, self.bias, self.talk, self.dim)
        return self.o_proj(o.reshape(x.shape[0], self.Hq * self.dim))


class DifferentialAttention(nn.Module):
    """Two attention maps per head over the same values: ``o = rms(a1 - lam a2) * (1 - diff)`` with a1, a2 the maps' outputs and one learned
    ``lam`` per layer. Queries and keys are laid out head by head as (map 1, map 2), each map normalised and rotated by itself; scores may be
    soft-capped, and attention may stay inside chunks of the sequence.

    fused QKV GEMM -> per-map norm, rotation and cache insert (one kernel) -> paged attention with both maps of a head in one CTA, which takes
    the difference and normalises it -> output projection. A cached key row holds both maps side by side."""

    kv_shared, window, window_keep, bias_table = False, 0, 0, None   # what the runner and the graphs ask of an attention layer

    def __init__(self, cfg: ModelConfig, layer_idx: int, prefix: str, device):
        super().__init__()
        tp = get_state().tp_size
        H, G = cfg.num_attention_heads, cfg.num_key_value_heads
        if H % tp or (G % tp and tp % G):
            raise ValueError(f"tensor_parallel_size={tp} does not divide the heads of layer {layer_idx}")
        self.dim, self.vdim = cfg.head_dim, cfg.v_head_dim or cfg.head_dim
        self.qkv_proj = QKVParallelLinear(cfg.hidden_size, 2 * self.dim, H, G, v_dim=self.vdim, quant=cfg.quant, prefix=prefix + ".qkv_proj",
                                          dtype=cfg.dtype)
        self.H, self.Hkv = self.qkv_proj.num_heads, self.qkv_proj.num_kv_heads
        self.Hq = 2 * self.H   # rows of the attention kernel: (head, map)
        self.o_proj = RowParallelLinear(H * self.vdim, cfg.hidden_size, quant=cfg.quant, prefix=prefix + ".o_proj", dtype=cfg.dtype)
        vec = lambda: nn.Parameter(torch.ones(self.dim, dtype=cfg.dtype), requires_grad=False)
        self.q_norm, self.k_norm = vec(), vec()
        self.lq1, self.lk1, self.lq2, self.lk2 = (nn.Parameter(torch.zeros(self.dim, dtype=torch.float32), requires_grad=False) for _ in range(4))
        self.register_buffer("lam", torch.zeros(1, dtype=torch.float32), persistent=False)
        self.diff, self.eps = cfg.attn_diff, cfg.rms_norm_eps
        self.rope = get_rope(cfg.rotary_dim, cfg.max_model_len, cfg.rope_theta, device, cfg.rope_scaling)
        self.scale = cfg.attn_scale if cfg.attn_scale is not None else cfg.head_dim ** -0.5
        self.softcap, self.chunk = cfg.attn_softcap, cfg.attn_chunk
        # width of a cached key (both maps) and value row: the next size of the tensor-core kernels
        need = max(2 * self.dim, self.vdim + self.vdim % 2)
        tc = torch.device(device).type == "cuda" and cfg.dtype == torch.bfloat16
        self.D = next((d for d in (64, 128, 256) if d >= need), need) if tc else need
        self.layer_idx = layer_idx

    def load_weight(self, pname: str, w: torch.Tensor, shard_id=None) -> None:
        getattr(self, pname).data.copy_(w)

    def process_weights_after_loading(self) -> None:
        lam = torch.exp((self.lq1.data * self.lk1.data).sum()) - torch.exp((self.lq2.data * self.lk2.data).sum()) + self.diff
        self.lam.copy_(lam)

    def forward(self, x: torch.Tensor, md, kv_cache: torch.Tensor) -> torch.Tensor:
        q = ops.diff_prepare(self.qkv_proj(x), self.q_norm, self.k_norm, self.eps, md.positions, self.rope.cos_sin, kv_cache, md.slot_mapping, self.H,
                             self.Hkv, self.dim, self.vdim)
        o = ops.diff_attention(q, kv_cache, md, self.scale, self.lam, 1.0 - self.diff, self.eps, self.vdim, self.softcap, self.chunk)
        return self.o_proj(o.reshape(x.shape[0], self.H * self.vdim))

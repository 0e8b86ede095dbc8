"""Op entry points. CUDA tensors go to the hand-written sm_100a kernels in the in-tree extension
(``onecat_vllm.ops.cuda``); CPU tensors go to the PyTorch restatements in ``onecat_vllm.ops.ref``.
There is no silent fallback: a CUDA tensor without the extension raises."""
from __future__ import annotations

from typing import Optional

import torch

from onecat_vllm.ops import ref

_ext = None


def ext():
    global _ext
    if _ext is None:
        from onecat_vllm.ops import cuda as _c
        _ext = _c
    return _ext


def rms_norm(x, w, eps, residual=None, gemma=False):
    if x.is_cuda:
        return ext().rms_norm(x, w, eps, residual, gemma)
    return ref.rms_norm(x, w, eps, residual, gemma)


def silu_and_mul(x):
    if x.is_cuda:
        return ext().silu_and_mul(x)
    return ref.silu_and_mul(x)


def gelu_tanh_and_mul(x):
    """GeGLU activation; an elementwise PyTorch expression on either device (Gemma-family models only)."""
    return ref.gelu_tanh_and_mul(x)


def rope_and_cache(q, k, v, positions, cos_sin, kv_cache, slot_mapping, rotary_dim, q_norm_w=None, k_norm_w=None,
                   eps=1e-6, gemma=False, mrope_section=None):
    """``mrope_section`` (three frequency counts summing to ``rotary_dim / 2``) with ``positions`` of shape ``[3, T]``: frequency i
    rotates by the temporal, height or width position according to the section it falls in (Qwen2-VL family)."""
    if q.is_cuda:
        return ext().rope_and_cache(q, k, v, positions, cos_sin, kv_cache, slot_mapping, rotary_dim, q_norm_w, k_norm_w, eps, gemma, mrope_section)
    return ref.rope_and_cache(q, k, v, positions, cos_sin, kv_cache, slot_mapping, rotary_dim, q_norm_w, k_norm_w, eps, gemma, mrope_section)


def kv_insert(k, kv_cache, slot_mapping, v=None):
    """Copy key (and value) rows into the paged cache, no rotation or norm (a cache with one tensor per page holds keys that are the values)."""
    if k.is_cuda:
        return ext().kv_insert(k, kv_cache, slot_mapping, v)
    return ref.kv_insert(k, kv_cache, slot_mapping, v)


def _norm_spec(norm):
    """(kind, weight, bias, eps, weight stored minus one, alpha) of a norm module: kind 1 RMS, 2 layer norm, 3 dynamic tanh."""
    if norm is None:
        return None
    alpha = getattr(norm, "alpha", None)
    kind = 3 if alpha is not None else 2 if getattr(norm, "plain", False) else 1
    return kind, norm.weight, getattr(norm, "bias", None), norm.eps, bool(norm.gemma), alpha


def stream_join(part, x, post, scale, nxt, out_dtype=None, add=None, copy_out=None, mul=1.0):
    """Join a sub-block's output to the fp32 residual stream and normalise it for the next one, in one kernel:
    ``x += mul * scale * post(part) (+ add)``, ``y = nxt(x)``. ``post`` / ``nxt`` are norm modules or None, ``scale`` a vector and ``mul`` a
    number. Returns (y, x); see ``ref.stream_join``."""
    f = ext().stream_join if part.is_cuda else ref.stream_join
    return f(part, x, _norm_spec(post), scale, _norm_spec(nxt), out_dtype, add, copy_out, mul)


def mla_prepare(q_latent, kv, q_norm, kv_norm, positions, cos_sin, cache, slot_mapping, lora, lora_pad, interleaved):
    """Latent attention between its down- and up-projections: the normalised query latent comes back (None without one), the normalised
    key/value latent and the rotated key part (``kv`` = [latent | key part]) go into the paged cache."""
    f = ext().mla_prepare if kv.is_cuda else ref.mla_prepare
    return f(q_latent, kv, q_norm.weight if q_norm is not None else None, kv_norm.weight, kv_norm.eps, positions, cos_sin, cache, slot_mapping, lora,
             lora_pad, interleaved)


def sigmoid_mul(x, gate):
    """``x * sigmoid(gate)`` element by element, both ``[T, n]`` (the gate may be a column slice)."""
    if x.is_cuda:
        return ext().sigmoid_mul(x, gate)
    return (x.float() * torch.sigmoid(gate.float())).to(x.dtype)


def embed_stream(ids, table, scale, prev=None, bigram=None, muls=(0, 0), out_dtype=None, gathered=False, rows=None, positions=None):
    """Scaled token embeddings plus hashed-bigram rows or learned position rows as the start of an fp32 residual stream; returns (stream, stream in ``out_dtype``).
    See ``ref.embed_stream``."""
    f = ext().embed_stream if table.is_cuda else ref.embed_stream
    return f(ids, table, scale, prev, bigram, muls, out_dtype or table.dtype, gathered, rows, positions)


def diff_prepare(qkv, q_norm, k_norm, eps, positions, cos_sin, kv_cache, slot_mapping, heads, kv_heads, dim, vdim, interleaved=True):
    """Norm, rotation and cache insert of differential attention's queries, keys and values in one kernel; returns the queries. See
    ``ref.diff_prepare``."""
    f = ext().diff_prepare if qkv.is_cuda else ref.diff_prepare
    return f(qkv, q_norm, k_norm, eps, positions, cos_sin, kv_cache, slot_mapping, heads, kv_heads, dim, vdim, interleaved)


def diff_attention(q, kv_cache, md, scale, lam, out_scale, eps, vdim, softcap=0.0, chunk=0):
    """Differential attention of the step ``md``: two softmax maps per head over the same values, their difference, the head norm. See
    ``ref.diff_attention``."""
    if q.is_cuda:
        return ext().diff_attention(q, kv_cache, md, scale, lam, out_scale, eps, vdim, softcap, chunk)
    return ref.diff_attention(q, kv_cache, md.block_table, md.query_start_loc, md.seq_lens, scale, lam, out_scale, eps, vdim, softcap, chunk)


def talk_prepare(qk, q_gain, eps, temperature, positions, pages, k_scale, slot_mapping, heads, kv_heads, dim):
    """Norm and temperature of talking-heads attention's queries, cache insert of its keys in one kernel; returns the queries. See
    ``ref.talk_prepare``."""
    f = ext().talk_prepare if qk.is_cuda else ref.talk_prepare
    return f(qk, q_gain, eps, temperature, positions, pages, k_scale, slot_mapping, heads, kv_heads, dim)


def talk_attention(q, pages, k_scale, md, bias, mix, dim):
    """Talking-heads attention of the step ``md`` with heads of ``dim`` columns; see ``ref.talk_attention``."""
    if q.is_cuda:
        return ext().talk_attention(q, pages, k_scale, md, bias, mix, dim)
    return ref.talk_attention(q, pages, k_scale, md.block_table, md.query_start_loc, md.seq_lens, bias, mix)


conv_state_shape = ref.conv_state_shape   # one slot of ``causal_conv``'s state


def causal_conv(x, weight, bias, state, md, silu=False, residual=False):
    """Causal convolution per channel over the step's portions with a rolling state; see ``ref.causal_conv``."""
    f = ext().causal_conv if x.is_cuda else ref.causal_conv
    return f(x, weight, bias, state, md, silu, residual)


def channel_delta(qkv, a, b, A_log, dt_bias, state, md, Hk, H, D, V):
    """Gated delta rule with one decay per key channel; see ``ref.channel_delta``."""
    f = ext().channel_delta if qkv.is_cuda else ref.channel_delta
    return f(qkv, a, b, A_log, dt_bias, state, md, Hk, H, D, V)


def mamba2(xbc, dt, A_log, dt_bias, D, state, md, H, G, N, V, dt_limit=(0.0, float("inf"))):
    """Mamba-2 state space; see ``ref.mamba2``."""
    f = ext().mamba2 if xbc.is_cuda else ref.mamba2
    return f(xbc, dt, A_log, dt_bias, D, state, md, H, G, N, V, dt_limit)


def gated_norm(x, gate, w, eps, groups, gate_first):
    """RMS norm in equal parts with a gate ahead of it (SiLU) or behind it (sigmoid); see ``ref.gated_norm``."""
    f = ext().gated_norm if x.is_cuda else ref.gated_norm
    return f(x, gate, w, eps, groups, gate_first)


def mlstm(qkvg, gates, i_bias, f_bias, norm_w, eps, cap, H, D, V, state, md):
    """mLSTM recurrence with its head norm and output gate: ``qkvg`` ``[T, 2 H D + 2 H V]`` (q | k | v | output gate), ``gates`` fp32
    ``[T, 2 H]`` (input | forget logits before bias and cap), ``state`` = (S, n, m) per slot, updated in place. Returns ``[T, H V]``."""
    f = ext().mlstm if qkvg.is_cuda else ref.mlstm
    return f(qkvg, gates, i_bias, f_bias, norm_w, eps, cap, H, D, V, state, md)


def paged_attention(q, kv_cache, md, scale, out=None, window=0, softcap=0.0, sinks=None, keep=0, bias_table=None, gate=None,
                    chunk=0):
    """``md`` is the step's AttentionMetadata. ``window``: sliding window in tokens (0 = full causal); ``softcap``: tanh soft-capping
    of the scaled scores (0 = off); ``sinks``: fp32 ``[Hq]`` sink logits that join the softmax denominator; ``keep``: first tokens visible
    outside the window; ``bias_table``: fp32 ``[Hq, n]`` added by distance; ``gate``: ``[T, Hq]`` logits of the per-head output gate;
    ``chunk``: only keys of the query's own chunk of that many positions are visible."""
    if q.is_cuda:
        return ext().paged_attention(q, kv_cache, md, scale, out, window=window, softcap=softcap, sinks=sinks, keep=keep, bias_table=bias_table,
                                     gate=gate, chunk=chunk)
    from onecat_vllm import envs
    extended = keep or bias_table is not None or gate is not None or kv_cache.shape[1] == 1 or chunk   # not in the native CPU kernel
    if envs.ONECAT_CPU_ATTENTION == "native" and not extended and kv_cache.dtype in (torch.float32, torch.bfloat16) and q.dtype in (torch.float32, torch.bfloat16):
        return cpu_paged_attention(q, kv_cache, md.block_table, md.query_start_loc, md.seq_lens, scale, out, window=window, softcap=softcap, sinks=sinks)
    return ref.paged_attention(q, kv_cache, md.block_table, md.query_start_loc, md.seq_lens, scale, out, window=window, softcap=softcap,
                               sinks=sinks, keep=keep, bias_table=bias_table, gate=gate, chunk=chunk)


def cpu_paged_attention(q, kv_cache, block_table, query_start_loc, seq_lens, scale, out=None, return_lse=False, window=0, softcap=0.0, sinks=None,
                        threads: int = 0):
    """The C++ paged attention of the CPU backend (``csrc/native/cpu_attention.cpp``): same contract as ``ref.paged_attention`` for fp32 /
    bf16 queries and caches."""
    from onecat_vllm.utils import _native
    T, Hq, D = q.shape
    if q.stride(2) != 1:
        q = q.contiguous()
    o = torch.empty(T, Hq, D, dtype=q.dtype) if out is None else out
    assert o.stride(2) == 1 and kv_cache.is_contiguous() and o.dtype == q.dtype
    lse = torch.full((T, Hq), -float("inf"), dtype=torch.float32) if return_lse else None
    bt = block_table if block_table.dtype == torch.int32 else block_table.to(torch.int32)
    qsl = query_start_loc.to(torch.int32).contiguous()
    sl = seq_lens.to(torch.int32).contiguous()
    sk = sinks.float().contiguous() if sinks is not None else None
    _native.cpu_paged_attention(q.data_ptr(), kv_cache.data_ptr(), o.data_ptr(), lse.data_ptr() if lse is not None else 0, bt.data_ptr(), qsl.data_ptr(),
                                sl.data_ptr(), sk.data_ptr() if sk is not None else 0, q.stride(0), q.stride(1), o.stride(0), o.stride(1), bt.stride(0),
                                sl.shape[0], Hq, kv_cache.shape[2], D, kv_cache.shape[3], float(scale), int(window), float(softcap),
                                int(q.dtype == torch.bfloat16), int(kv_cache.dtype == torch.bfloat16), int(threads))
    return (o, lse) if return_lse else o


def rms_norm_gated(x, z, w, eps, heads):
    """x, z ``[T, heads*D]`` (column slices allowed) → ``[T, heads*D]``: per-head RMSNorm(x) * w * silu(z)."""
    if x.is_cuda:
        return ext().rms_norm_gated(x, z, w, eps, heads)
    T, D = x.shape[0], x.shape[1] // heads
    return ref.rms_norm_gated(x.reshape(T * heads, D), z.reshape(T * heads, D), w, eps).reshape(T, heads * D)


def merge_attn_states(o1, lse1, o2, lse2):
    """LSE-weighted merge of two partial attention results over disjoint key sets."""
    if o1.is_cuda:
        return ext().merge_attn_states(o1, lse1, o2, lse2)
    return ref.merge_attn_states(o1, lse1, o2, lse2)


def argmax(logits):
    if logits.is_cuda:
        return ext().argmax(logits)
    return logits.argmax(-1)

"""Python side of the sm_100a kernels: weight repacking, workspaces, launch planning.

Importing this module loads the in-tree extension ``onecat_vllm.ops._C`` and fails loudly when it is missing: on a
CUDA device there is no eager fallback for the ops implemented here. Ops whose kernels are not written yet
(listed in ``TORCH_STANDINS``) run the PyTorch restatement on the device and are reported as such."""
from __future__ import annotations

import os
from typing import Optional

import torch

from onecat_vllm.ops import ref

try:
    from onecat_vllm.ops import _C
except ImportError as e:  # pragma: no cover
    raise ImportError("the CUDA extension onecat_vllm.ops._C is not built; run `python -c 'import __graft_entry__ as g; g.build()'` "
                      f"or `python 1cat-vllm_b200/ops/build.py` ({e})") from e

EPI_STORE, EPI_SILU_MUL, EPI_GELU_TANH, EPI_GELU_MUL = 0, 1, 2, 3
TORCH_STANDINS: set = set()  # names of ops that ran as device-side PyTorch code in this process
_LAUNCHES = 0  # launches of our own kernels (for bench accounting)
_LIB_GEMM = os.environ.get("ONECAT_GEMM_BACKEND", "tcgen05") == "library"  # debug switch only
_ATTN_PREFILL_TC = os.environ.get("ONECAT_ATTN_PREFILL", "tcgen05") != "mma"  # head size 128 prefill: tcgen05 kernel unless "mma"


def launches() -> int:
    return _LAUNCHES


def reset_launches() -> None:
    global _LAUNCHES
    _LAUNCHES = 0


class _Workspace:
    """Per-device scratch: split-K partials + tile counters, split-KV partials."""

    def __init__(self, device):
        self.device = device
        self.splitk = torch.empty(64 << 20, dtype=torch.uint8, device=device)
        self.counters = torch.zeros(8192, dtype=torch.int32, device=device)  # upper half: scratch
        self.attn_o = None
        self.attn_ml = None

    def attn_static(self, n_o: int, n_ml: int):
        """Buffers whose addresses are baked into CUDA graphs: sized once per engine for its largest graph."""
        if getattr(self, "s_o", None) is None or self.s_o.numel() < n_o or self.s_ml.numel() < n_ml:
            # a later engine in the same process may need more; graphs captured earlier keep their (retired) buffers alive
            if getattr(self, "s_o", None) is not None:
                self._retired = getattr(self, "_retired", []) + [(self.s_o, self.s_ml)]
            self.s_o = torch.empty(n_o, dtype=torch.float32, device=self.device)
            self.s_ml = torch.empty(n_ml, dtype=torch.float32, device=self.device)
        return self.s_o, self.s_ml

    def attn(self, n_o: int, n_ml: int):
        if self.attn_o is None or self.attn_o.numel() < n_o:
            self.attn_o = torch.empty(n_o, dtype=torch.float32, device=self.device)
        if self.attn_ml is None or self.attn_ml.numel() < n_ml:
            self.attn_ml = torch.empty(n_ml, dtype=torch.float32, device=self.device)
        return self.attn_o, self.attn_ml


_WS: dict = {}


def workspace(device) -> _Workspace:
    key = device.index if device.index is not None else torch.cuda.current_device()
    if key not in _WS:
        _WS[key] = _Workspace(torch.device("cuda", key))
    return _WS[key]


def check_status(clear: bool = True) -> int:
    return int(_C.read_status(clear))


# ----------------------------------------------------------------------------- weight repacking
_NIB_ORDER = (0, 2, 4, 6, 1, 3, 5, 7)  # nibble i of a packed word holds k offset _NIB_ORDER[i]


def interleave_gate_up(n_inter: int, device) -> torch.Tensor:
    """Row permutation putting 16 gate rows next to the matching 16 up rows, so that one warp of the GEMM epilogue
    holds both halves of SiLU(gate)*up."""
    assert n_inter % 16 == 0, "the intermediate size must be a multiple of 16"
    b = torch.arange(n_inter // 16, device=device).view(-1, 1, 1) * 16
    j = torch.arange(16, device=device).view(1, 1, 16)
    half = torch.tensor([0, n_inter], device=device).view(1, 2, 1)
    return (b + j + half).reshape(-1)


def pack_w4(q: torch.Tensor, z: torch.Tensor, s: torch.Tensor, group: int):
    """q ``[N,K]`` uint8 codes, z ``[N,K/g]`` uint8 zeros, s ``[N,K/g]`` scales → (tiles uint8 ``[N/128, K/64, 4096]``,
    sz int32 ``[K/g, Npad]``). A tile holds 128 rows × 64 k as two halves of ``[128 rows][4 words]``; each 32-bit word is
    8 consecutive k of one row in ``_NIB_ORDER``."""
    N, K = q.shape
    assert K % 64 == 0 and group % 64 == 0, "K and the group size must be multiples of 64"
    npad = -(-N // 128) * 128
    if npad != N:
        q = torch.cat([q, q.new_zeros(npad - N, K)])
        z = torch.cat([z, z.new_zeros(npad - N, z.shape[1])])
        s = torch.cat([s, s.new_zeros(npad - N, s.shape[1])])
    nt, kt = npad // 128, K // 64
    qq = q.view(nt, 128, kt, 8, 8).to(torch.int32)
    words = torch.zeros(nt, 128, kt, 8, dtype=torch.int32, device=q.device)
    for i, k in enumerate(_NIB_ORDER):
        words |= qq[..., k] << (4 * i)
    tiles = words.view(nt, 128, kt, 2, 4).permute(0, 2, 3, 1, 4).contiguous().view(torch.uint8).view(nt, kt, 4096)
    sb = s.to(torch.bfloat16).view(torch.int16).to(torch.int32) & 0xFFFF
    zb = (z.to(torch.float32) + 128.0).to(torch.bfloat16).view(torch.int16).to(torch.int32) & 0xFFFF
    sz = (sb | (zb << 16)).t().contiguous()
    return tiles, sz, npad


def prepare_w4(layer, q: torch.Tensor, z: torch.Tensor, s: torch.Tensor, group: int) -> None:
    """Repack a 4-bit layer for the kernel. ``q/z/s`` are in logical ``[out, in]`` orientation."""
    n_rows = q.shape[0]
    n_out = n_rows
    epi = EPI_STORE
    if layer.fuse_silu_mul:
        perm = interleave_gate_up(n_rows // 2, q.device)
        q, z, s = q[perm], z[perm], s[perm]
        n_out, epi = n_rows // 2, EPI_SILU_MUL
    tiles, sz, npad = pack_w4(q.contiguous(), z.contiguous(), s.contiguous(), group)
    layer.kernel_state = dict(kind="w4", tiles=tiles, sz=sz, n_rows=n_rows, n_out=n_out, n_pad=npad, epi=epi, group_ktiles=group // 64,
                              K=q.shape[1])


def prepare_bf16(layer) -> None:
    w = layer.weight.data
    n_rows, epi, n_out = w.shape[0], EPI_STORE, w.shape[0]
    gelu_mul = getattr(layer, "fuse_gelu_mul", False)
    if layer.fuse_silu_mul or gelu_mul:
        n = n_rows // 2
        if n % 16:   # the epilogue pairs 16 gate rows with 16 up rows: zero rows make up the last block (their outputs are cut off)
            w = torch.nn.functional.pad(w.view(2, n, -1), (0, 0, 0, -n % 16)).reshape(-1, w.shape[1])
            n_rows = w.shape[0]
        w = w[interleave_gate_up(n_rows // 2, w.device)].contiguous()
        layer.weight.data = w
        epi, n_out = EPI_GELU_MUL if gelu_mul else EPI_SILU_MUL, n_rows // 2
    elif getattr(layer, "fuse_gelu_tanh", False):
        epi = EPI_GELU_TANH
    layer.kernel_state = dict(kind="bf16", n_rows=n_rows, n_out=n_out, epi=epi, K=w.shape[1])
    if epi in (EPI_SILU_MUL, EPI_GELU_MUL) and n != n_out:
        layer.kernel_state["n_cut"] = n
    if w.shape[1] % 64:   # the GEMM walks whole 64-wide k tiles: zero columns in a copy that only the kernel reads
        layer.kernel_state["w_pad"] = torch.nn.functional.pad(w, (0, -w.shape[1] % 64)).contiguous()


def _bf16_bits(x: torch.Tensor) -> torch.Tensor:
    return x.to(torch.bfloat16).view(torch.int16).to(torch.int32) & 0xFFFF


def pack_fp8(w8: torch.Tensor, row_scale: torch.Tensor, group: int):
    """w8 ``[N,K]`` e4m3 (any 1-byte dtype), row_scale ``[N, K/group]`` fp32 (dequantisation scale of each row over each k group;
    group a multiple of 64) → (tiles uint8 ``[N/128, K/64, 8192]``, sz int32 ``[K/group, Npad]``). A tile is four chunks of
    ``[128 rows][16 bytes]`` (chunk c = k 16c..16c+15); the scale words are ``bf16(scale * 2**120)``: the kernel builds each bf16
    from the fp8 bits with the exponent 120 too small."""
    N, K = w8.shape
    assert K % 64 == 0 and group % 64 == 0 and K % group == 0
    npad = -(-N // 128) * 128
    w8 = w8.contiguous().view(torch.uint8)
    if npad != N:
        w8 = torch.cat([w8, w8.new_zeros(npad - N, K)])
        row_scale = torch.cat([row_scale, row_scale.new_zeros(npad - N, row_scale.shape[1])])
    nt, kt = npad // 128, K // 64
    tiles = w8.view(nt, 128, kt, 4, 16).permute(0, 2, 3, 1, 4).contiguous().view(nt, kt, 8192)
    sc = row_scale.float() * (2.0 ** 120)
    assert bool(torch.isfinite(sc.to(torch.bfloat16)).all()), "fp8 scale too large for the bf16 scale word"
    sz = _bf16_bits(sc).t().contiguous()
    return tiles, sz, npad


def pack_mxfp4(packed: torch.Tensor, scales_ue8m0: torch.Tensor):
    """packed ``[N, K/2]`` uint8 (low nibble = even k), scales ``[N, K/32]`` ue8m0 → (tiles uint8 ``[N/128, K/64, 4096]`` in the
    4-bit tile layout of ``pack_w4``, sz int32 ``[K/64, Npad]`` with the two 32-k groups' ``bf16(2**(e-127) * 2**126)`` in the low
    and high half)."""
    N, K2 = packed.shape
    K = K2 * 2
    assert K % 64 == 0
    npad = -(-N // 128) * 128
    q = torch.stack([packed & 0xF, packed >> 4], dim=-1).reshape(N, K)
    e = scales_ue8m0.to(torch.int32)
    if npad != N:
        q = torch.cat([q, q.new_zeros(npad - N, K)])
        e = torch.cat([e, e.new_full((npad - N, e.shape[1]), 127)])
    nt, kt = npad // 128, K // 64
    qq = q.view(nt, 128, kt, 8, 8).to(torch.int32)
    words = torch.zeros(nt, 128, kt, 8, dtype=torch.int32, device=q.device)
    for i, k in enumerate(_NIB_ORDER):
        words |= qq[..., k] << (4 * i)
    tiles = words.view(nt, 128, kt, 2, 4).permute(0, 2, 3, 1, 4).contiguous().view(torch.uint8).view(nt, kt, 4096)
    assert int(e.max()) <= 128, "MXFP4 scale above 2.0 does not fit the bf16 scale word"
    sb = _bf16_bits(torch.exp2(e.float() - 1.0)).view(npad, kt, 2)
    sz = (sb[..., 0] | (sb[..., 1] << 16)).t().contiguous()
    return tiles, sz, npad


def pack_nvfp4(packed: torch.Tensor, scales_e4m3: torch.Tensor, global_scale: torch.Tensor):
    """packed ``[N, K/2]`` uint8 (low nibble = even k), scales ``[N, K/16]`` e4m3, one fp32 global scale → (tiles as ``pack_mxfp4``,
    sz int32 ``[K/64, Npad, 2]``: per row and k tile the four 16-k groups' ``bf16(scale * global * 2**126)``, two per word)."""
    N, K2 = packed.shape
    K = K2 * 2
    assert K % 64 == 0
    tiles, _, npad = pack_mxfp4(packed, torch.full((N, K // 32), 127, dtype=torch.uint8, device=packed.device))
    sc = scales_e4m3.float() * global_scale.float().reshape(-1)[0] * (2.0 ** 126)
    assert bool(torch.isfinite(sc.to(torch.bfloat16)).all()), "NVFP4 scale too large for the bf16 scale word"
    if npad != N:
        sc = torch.cat([sc, sc.new_zeros(npad - N, sc.shape[1])])
    sb = _bf16_bits(sc).view(npad, K // 64, 2, 2)
    sz = (sb[..., 0] | (sb[..., 1] << 16)).permute(1, 0, 2).contiguous()
    return tiles, sz, npad


def _fp8_row_scales(layer, block) -> tuple[torch.Tensor, int]:
    """Per-row, per-k-group dequantisation scales of an FP8 linear layer and the k group size."""
    N, K = layer.weight.shape
    if block:
        bn, bk = block
        assert bk % 64 == 0, "fp8 k blocks must be multiples of 64"
        return layer.weight_scale_inv.float().repeat_interleave(bn, dim=0)[:N].contiguous(), bk
    ws = layer.weight_scale.float().reshape(-1)
    if ws.numel() == N and getattr(layer.method, "channel", False):
        return ws.reshape(N, 1).contiguous(), K   # one scale per output channel
    if ws.numel() == 1:
        return ws.expand(N).reshape(N, 1).contiguous(), K
    rows = torch.cat([ws[i].expand(n) for i, n in enumerate(layer.local_output_sizes)])
    return rows.reshape(N, 1).contiguous(), K


def prepare_fp8(layer, block) -> None:
    """FP8 e4m3 weights stay one byte each in HBM: tiles + scale words for the weight-only path of the tcgen05 GEMM
    (dequantised to bf16 on the way into TMEM; activations stay bf16)."""
    N, K = layer.weight.shape
    if K % 64 or (block and (K % block[1] or block[1] % 64)):
        w = layer.method.dequantized_weight(layer).to(torch.bfloat16)
        return _swap_to_dense(layer, w)
    rs, group = _fp8_row_scales(layer, block)
    w8 = layer.weight.data
    n_rows, n_out, epi = N, N, EPI_STORE
    if layer.fuse_silu_mul:
        perm = interleave_gate_up(N // 2, w8.device)
        w8, rs = w8.view(torch.uint8)[perm], rs[perm]
        n_out, epi = N // 2, EPI_SILU_MUL
    tiles, sz, npad = pack_fp8(w8, rs, group)
    layer.kernel_state = dict(kind="w4", wkind=2, tiles=tiles, sz=sz, n_rows=n_rows, n_out=n_out, n_pad=npad, epi=epi, group_ktiles=group // 64, K=K)
    for n in ("weight", "weight_scale", "weight_scale_inv"):
        if hasattr(layer, n):
            delattr(layer, n)


def prepare_fp4(layer, kind: str) -> None:
    """MXFP4 and NVFP4 weights stay packed (tiles + scale words, dequantised to bf16 on the way into TMEM)."""
    N, K2 = layer.weight.shape
    if kind not in ("mxfp4", "nvfp4") or (K2 * 2) % 64:
        w = layer.method.dequantized_weight(layer).to(torch.bfloat16)
        return _swap_to_dense(layer, w)
    pk, sc = layer.weight.data, layer.weight_scale.data
    n_rows, n_out, epi = N, N, EPI_STORE
    if layer.fuse_silu_mul:
        perm = interleave_gate_up(N // 2, pk.device)
        pk, sc = pk[perm], sc[perm]
        n_out, epi = N // 2, EPI_SILU_MUL
    if kind == "nvfp4":
        tiles, sz, npad = pack_nvfp4(pk.contiguous(), sc.contiguous(), layer.weight_scale_2.data)
    else:
        tiles, sz, npad = pack_mxfp4(pk.contiguous(), sc.contiguous())
    layer.kernel_state = dict(kind="w4", wkind=4 if kind == "nvfp4" else 3, tiles=tiles, sz=sz, n_rows=n_rows, n_out=n_out, n_pad=npad, epi=epi,
                              group_ktiles=1, K=K2 * 2)
    for n in ("weight", "weight_scale", "weight_scale_2"):
        if hasattr(layer, n):
            delattr(layer, n)


def _swap_to_dense(layer, w: torch.Tensor) -> None:
    from onecat_vllm.layers.linear import UnquantizedMethod
    for n in ("weight", "weight_scale", "weight_scale_inv", "weight_scale_2"):
        if hasattr(layer, n):
            delattr(layer, n)
    layer.weight = torch.nn.Parameter(w.contiguous(), requires_grad=False)
    layer.method = UnquantizedMethod()
    prepare_bf16(layer)


# ----------------------------------------------------------------------------- GEMM
def _gemm(x, w, w4, sz, out, bias, N, n_rows, n_out, n_pad, epi, gk, force_splits=0, force_tn=0, push=None, wkind=1, trace=0):
    """``push`` = (list of destination addresses, rows per owner[, address of the buffer-select word, buffer stride in elements]):
    tensor-parallel epilogue that stores into peers' slabs (the last two for the flag-free arrival buffers)."""
    global _LAUNCHES
    ws = workspace(x.device)
    _C.gemm(x, w, w4, sz, out, bias, ws.splitk, ws.counters, N, n_rows, n_out, n_pad, epi, gk, force_splits, force_tn,
            push[0] if push else [], push[1] if push else 0, wkind if w4 is not None else 0, trace,
            push[2] if push and len(push) > 2 else 0, push[3] if push and len(push) > 2 else 0)
    _LAUNCHES += 1
    return out


def gemm_bf16(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
              force_splits: int = 0, force_tn: int = 0, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """x ``[T,K]`` @ w ``[N,K]``^T → ``[T,N]`` bf16, or fp32 (the accumulators) with ``out_dtype``."""
    N = w.shape[0]
    if _LIB_GEMM:
        y = torch.nn.functional.linear(x, w, bias)
        return y if out_dtype is None else y.to(out_dtype)
    if x.shape[1] % 64:
        x, w = (torch.nn.functional.pad(t, (0, -x.shape[1] % 64)) for t in (x, w))
    if out is None:
        out = torch.empty(x.shape[0], N, dtype=out_dtype or torch.bfloat16, device=x.device)
    if x.stride(-1) != 1 or (x.stride(0) * 2) % 16 or x.data_ptr() % 16:
        x = x.contiguous()
    return _gemm(x, w, None, None, out, bias, N, N, N, 0, EPI_STORE, 1, force_splits, force_tn)


def dense(x: torch.Tensor, w: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """x @ w^T in the inputs' precision: the tcgen05 GEMM for bf16, the library's fp32 product (no reduced-precision mode) for fp32."""
    if x.dtype == torch.float32:
        return _matmul_f32(x, w)
    return gemm_bf16(x, w, out_dtype=out_dtype)


def _matmul_f32(x, w, bias=None):
    if torch.backends.cuda.matmul.allow_tf32:
        raise RuntimeError("fp32 models need torch.backends.cuda.matmul.allow_tf32 = False")
    return torch.nn.functional.linear(x, w, bias)


def _linear_f32(layer, x: torch.Tensor) -> torch.Tensor:
    """Linear layer of an engine that runs in 32 bits (dense weights)."""
    global _LAUNCHES
    w = getattr(layer, "weight", None)
    if w is None or w.dtype != torch.float32:
        raise ValueError("quantised weights are served with bf16 activations only")
    y = _matmul_f32(x, w, layer.bias)
    if layer.fuse_silu_mul:
        return ref.silu_and_mul(y)
    if getattr(layer, "fuse_gelu_tanh", False):
        _LAUNCHES += 1
        _C.gelu_tanh_f32(y)
    if getattr(layer, "fuse_gelu_mul", False):
        return ref.gelu_tanh_and_mul(y)
    return y


def linear(layer, x: torch.Tensor, out: Optional[torch.Tensor] = None, push=None) -> torch.Tensor:
    if x.dtype == torch.float32:
        return _linear_f32(layer, x)
    ks = layer.kernel_state
    if ks is None:
        prepare_bf16(layer)
        ks = layer.kernel_state
    T = x.shape[0]
    w = ks.get("w_pad")
    if w is not None:
        x = torch.nn.functional.pad(x, (0, w.shape[1] - x.shape[1]))
    if x.stride(-1) != 1 or (x.stride(0) * 2) % 16 or x.data_ptr() % 16:
        x = x.contiguous()
    if out is None:
        n = ks["n_out"]   # row pitches are multiples of 16 bytes, so that column slices of the result are aligned for the next kernel
        out = torch.empty(T, -(-n // 8) * 8, dtype=getattr(layer, "out_dtype", None) or torch.bfloat16, device=x.device)[:, :n]
    bias = layer.bias
    if ks["kind"] == "w4":
        if _LIB_GEMM:
            raise RuntimeError("the library GEMM debug switch does not cover 4-bit weights")
        y = _gemm(x, None, ks["tiles"], ks["sz"], out, bias, ks["n_rows"], ks["n_rows"], ks["n_out"], ks["n_pad"], ks["epi"], ks["group_ktiles"], push=push,
                  wkind=ks.get("wkind", 1))
        return torch.nn.functional.gelu(y, approximate="tanh") if getattr(layer, "fuse_gelu_tanh", False) else y
    if _LIB_GEMM:
        y = torch.nn.functional.linear(x, layer.weight if w is None else w, bias)
        if ks["epi"] == EPI_SILU_MUL:  # rows are interleaved in blocks of 16
            y = y.view(T, -1, 2, 16)
            return (torch.nn.functional.silu(y[:, :, 0].float()) * y[:, :, 1].float()).to(x.dtype).reshape(T, -1)[:, : ks.get("n_cut")]
        if ks["epi"] == EPI_GELU_MUL:
            y = y.view(T, -1, 2, 16)
            return (torch.nn.functional.gelu(y[:, :, 0].float(), approximate="tanh") * y[:, :, 1].float()).to(x.dtype).reshape(T, -1)[:, : ks.get("n_cut")]
        if ks["epi"] == EPI_GELU_TANH:
            y = torch.nn.functional.gelu(y, approximate="tanh")
        return y.to(out.dtype)
    y = _gemm(x, layer.weight if w is None else w, None, None, out, bias, ks["n_rows"], ks["n_rows"], ks["n_out"], 0, ks["epi"], 1, push=push)
    return y[:, : ks["n_cut"]] if "n_cut" in ks else y


# ----------------------------------------------------------------------------- elementwise
def rms_norm(x, w, eps, residual=None, gemma=False):
    global _LAUNCHES
    _LAUNCHES += 1
    if w.dtype != torch.bfloat16:
        w = w.to(torch.bfloat16)
    if x.stride(-1) != 1:
        x = x.contiguous()
    y, r = _C.rms_norm(x, w, eps, residual, gemma)
    return y, r


def rms_norm_gated(x, z, w, eps, heads):
    global _LAUNCHES
    _LAUNCHES += 1
    T = x.shape[0]
    if x.stride(-1) != 1:
        x = x.contiguous()
    if z.stride(-1) != 1:
        z = z.contiguous()
    return _C.rms_norm_gated(x, z, w.to(torch.bfloat16), eps, heads).view(T, -1)


def silu_and_mul(x):
    global _LAUNCHES
    _LAUNCHES += 1
    return _C.silu_and_mul(x.contiguous())


def rope_and_cache(q, k, v, positions, cos_sin, kv_cache, slot_mapping, rotary_dim, q_norm_w, k_norm_w, eps, gemma, mrope_section=None):
    global _LAUNCHES
    _LAUNCHES += 1
    s0, s1 = (int(mrope_section[0]), int(mrope_section[0] + mrope_section[1])) if mrope_section is not None and positions.dim() == 2 else (0, 0)
    _C.rope_and_cache(q, k, v, positions, cos_sin, kv_cache, slot_mapping, rotary_dim, q_norm_w, k_norm_w, eps, gemma, 1.0, 1.0, s0, s1)


def kv_insert(k, kv_cache, slot_mapping, v=None):
    global _LAUNCHES
    _LAUNCHES += 1
    _C.kv_insert(k, v, kv_cache, slot_mapping)


def stream_join(part, x, post, scale, nxt, out_dtype=None, add=None, copy_out=None, mul=1.0):
    global _LAUNCHES
    _LAUNCHES += 1
    T, H = part.shape
    x_out = torch.empty(T, H, dtype=torch.float32, device=part.device) if x is None else x
    y = torch.empty(T, H, dtype=out_dtype, device=part.device) if nxt is not None else None
    none = (0, None, None, 0.0, False, None)
    post, nxt = (tuple(n) + (None,) if len(n) == 5 else n for n in (post or none, nxt or none))
    _C.stream_join(part, x, x_out, *post[:5], scale, *nxt[:5], y, add, copy_out, (copy_out.dtype if y is None and copy_out is not None
                   else out_dtype or part.dtype) == torch.float32, mul, post[5], nxt[5])
    return y, x_out


def embed_stream(ids, table, scale, prev, bigram, muls, out_dtype, gathered=False, rows=None, positions=None):
    global _LAUNCHES
    _LAUNCHES += 1
    T, H = ids.shape[0], table.shape[1]
    x = torch.empty(T, H, dtype=torch.float32, device=table.device)
    y = torch.empty(T, H, dtype=out_dtype, device=table.device) if out_dtype != torch.float32 and rows is None else None
    _C.embed_stream(ids.to(torch.int32).contiguous(), table, scale, prev, bigram, muls[0], muls[1], x, y, gathered, rows,
                    positions)
    return x, (x if y is None else y)


def diff_prepare(qkv, q_norm, k_norm, eps, positions, cos_sin, kv_cache, slot_mapping, heads, kv_heads, dim, vdim, interleaved):
    global _LAUNCHES
    _LAUNCHES += 1
    return _C.diff_prepare(qkv if qkv.stride(-1) == 1 else qkv.contiguous(), q_norm, k_norm, eps, positions, cos_sin, kv_cache, slot_mapping, heads,
                           kv_heads, dim, vdim, interleaved)


def sample(logits, temperature, top_k=None, top_p=None, min_p=None, generators=None, kept=None):
    """One kernel per batch: temperature, min-p, top-k, top-p and the random draw (rows with temperature ~ 0 take their arg-max).
    Each row gets a 64-bit word of randomness: from its request's generator when it has one (so seeded requests repeat), else from
    the device's default generator."""
    global _LAUNCHES
    _LAUNCHES += 2
    B = logits.shape[0]
    seeds = torch.randint(0, 1 << 62, (B,), dtype=torch.int64, device=logits.device)
    for i, gen in (generators or {}).items():
        seeds[i] = torch.randint(0, 1 << 62, (1,), dtype=torch.int64, device=logits.device, generator=gen)[0]
    return _C.sample(logits, temperature.float().contiguous(), None if top_k is None else top_k.to(torch.int32).contiguous(),
                     None if top_p is None else top_p.float().contiguous(), None if min_p is None else min_p.float().contiguous(), seeds, kept)


def merge_attn_states(o1, lse1, o2, lse2):
    global _LAUNCHES
    _LAUNCHES += 1
    o, lse = _C.merge_attn_states(o1.contiguous(), lse1.float().contiguous(), o2.contiguous(), lse2.float().contiguous())
    return o, lse


def argmax(logits):
    global _LAUNCHES
    _LAUNCHES += 1
    return _C.argmax(logits)


# ----------------------------------------------------------------------------- attention
_NUM_SMS: dict = {}


def _sms(device) -> int:
    k = device.index or 0
    if k not in _NUM_SMS:
        _NUM_SMS[k] = torch.cuda.get_device_properties(device).multi_processor_count
    return _NUM_SMS[k]


def choose_kv_splits(base_ctas: int, max_seq: int, num_sms: int) -> int:
    """KV splits of the decode kernel: enough CTAs for about two full waves (two CTAs fit per SM), but at least four
    64-key tiles per split so that the copy pipeline fills."""
    want = -(-(4 * num_sms) // max(base_ctas, 1))
    by_ctx = max(1, -(-max_seq // 64) // 4)
    return max(1, min(want, by_ctx, 32))


def choose_decode_splits(base_ctas: int, max_seq: int, num_sms: int, per_sm: int = 2) -> int:
    """KV splits of the paged decode kernel from a cost model of its waves. ``per_sm`` CTAs fit per SM; a CTA needs about 1.6 us to start
    and 1.9 us per 64-key tile when the SMs are full, and more than one split adds the combine launch (about 6 us). Measured on
    B200 (64 requests x 8 KV heads x 1150 keys): 71.7 us unsplit against 80.9 us in two splits, whose 1024 CTAs need four waves
    of 296 where 512 need two; 16 requests x 4096 keys: 66 us in two splits (one wave) against 83 us in three (two waves)."""
    nt = max(1, -(-max_seq // 64))
    slots = per_sm * num_sms
    best, best_cost = 1, None
    for s in range(1, min(32, nt) + 1):
        per = -(-nt // s)
        if s > 1 and per < 2:
            break
        waves = -(-(max(base_ctas, 1) * s) // slots)
        cost = waves * (1.6 + 1.9 * per) + (6.0 + 0.15 * s if s > 1 else 0.0)  # the combine kernel reads one partial per split
        if best_cost is None or cost < best_cost - 1e-9:
            best, best_cost = s, cost
    return best


def plan_attention(query_lens: list, seq_lens: list, Hq: int, Hkv: int, D: int, num_sms: int, force_splits: int = 0, span: int = 0,
                   extended: bool = False):
    """Decide which requests take the decode kernel (rows = q_len * group fit in one 16/32-row tile) and how many KV
    splits it uses. Returns (short_q_len, num_q_tiles for the prefill kernel, splits). ``span`` > 0: a decode row reads at most that many
    keys of its context (window and kept first tokens). ``extended``: the variants of the kernel with one ring of shared keys and values,
    of which more CTAs fit per SM."""
    G = Hq // Hkv
    max_rows = 32 if D <= 128 else 16
    short = max_rows // G
    n_short = sum(1 for q in query_lens if 0 < q <= short)
    if n_short:  # the row tile of the decode kernel follows the longest short query actually present (q=1 -> 16 rows)
        short = max(q for q in query_lens if 0 < q <= short)
    TQ = 64 // G
    tiles = sum(-(-q // TQ) for q in query_lens if q > short)
    splits = 1
    if n_short:
        max_s = max((s for q, s in zip(query_lens, seq_lens) if q <= short), default=1)
        per_sm = {64: 5, 128: 4}.get(D, 2) if extended and short * G <= 16 else 2
        splits = choose_decode_splits(n_short * Hkv, min(max_s, span) if span else max_s, num_sms, per_sm)
    if force_splits:
        splits = force_splits
    return short, tiles, splits


def attention_span(window: int, keep: int) -> int:
    """Most keys that the decode kernel walks for a sliding-window (or chunked) layer, in whole 64-key tiles; 0: the whole context."""
    return 64 * (-(-window // 64) + 1 + -(-keep // 64)) if window else 0


def paged_attention(q, kv_cache, md, scale, out=None, lse=None, window=0, softcap=0.0, sinks=None, keep=0, bias_table=None, gate=None, chunk=0):
    """``window`` (tokens, 0 = full), ``softcap`` (0 = off), ``sinks`` (fp32 ``[Hq]``), ``keep`` (first tokens visible outside the window),
    ``bias_table`` (fp32 ``[Hq, n]`` by distance), ``gate`` (``[T, Hq]`` logits), ``chunk`` (positions, 0 = off) and a cache with one tensor per page select the mma.sync
    kernels; the tcgen05 prefill kernel serves plain causal attention with D = 128. fp32 queries run the fp32 kernel."""
    global _LAUNCHES
    T, Hq, D = q.shape
    Hkv = kv_cache.shape[2]
    if out is None:
        out = torch.empty(T, Hq, D, dtype=q.dtype, device=q.device)
    if q.dtype == torch.float32:
        G = Hq // Hkv
        tiles = sum(-(-n * G // 16) for n in md.query_lens_cpu)
        _C.paged_attention(q, kv_cache, out, lse, md.query_start_loc, md.seq_lens, md.block_table, scale, 3, tiles, 1, md.max_query_len, 0, None, None,
                           window, softcap, sinks, 1.0, 1.0, keep, bias_table, gate, chunk)
        _LAUNCHES += 1
        return out
    extended = keep > 0 or bias_table is not None or gate is not None or kv_cache.shape[1] == 1 or chunk > 0
    key = (Hq, Hkv, D, attention_span(min(window, chunk) if window and chunk else window or chunk, keep)) if extended else (Hq, Hkv, D)
    plan = getattr(md, "attn_plan", None)
    if plan is None or plan[0] != key:
        plan = (key, plan_attention(md.query_lens_cpu, md.seq_lens_cpu, Hq, Hkv, D, _sms(q.device), span=key[3] if extended else 0,
                                    extended=kv_cache.shape[1] == 1))
        md.attn_plan = plan
    short, tiles, splits = plan[1]
    n_short = sum(1 for x in md.query_lens_cpu if 0 < x <= short)
    ws_o = ws_ml = None
    if n_short and splits > 1:
        w = workspace(q.device)
        ws_o, ws_ml = (w.attn_static if getattr(md, "static_ws", False) else w.attn)(splits * T * Hq * D, splits * T * Hq * 2)
    if n_short:
        _C.paged_attention(q, kv_cache, out, lse, md.query_start_loc, md.seq_lens, md.block_table, scale, 1, 0, splits,
                           md.max_query_len, short, ws_o, ws_ml, window, softcap, sinks, 1.0, 1.0, keep, bias_table, gate, chunk)
        _LAUNCHES += 2 if splits > 1 else 1
    if tiles:
        if (D == 128 and q.stride(1) == D and _ATTN_PREFILL_TC and not window and not softcap and sinks is None and not extended
                and kv_cache.dtype == torch.bfloat16):
            # tcgen05 kernel: 128-token query tiles per (request, head)
            tiles_tc = sum(-(-x // 128) for x in md.query_lens_cpu if x > short)
            _C.paged_attention(q, kv_cache, out, lse, md.query_start_loc, md.seq_lens, md.block_table, scale, 2, tiles_tc, 1,
                               md.max_query_len, short, None, None, 0, 0.0, None, 1.0, 1.0)
        else:
            _C.paged_attention(q, kv_cache, out, lse, md.query_start_loc, md.seq_lens, md.block_table, scale, 0, tiles, 1,
                               md.max_query_len, short, None, None, window, softcap, sinks, 1.0, 1.0, keep, bias_table, gate, chunk)
        _LAUNCHES += 1
    return out


DIFF_PREFILL_MIN_LEN = 64          # a step with a portion of at least this many tokens runs its portions on tcgen05


def diff_attention(q, kv_cache, md, scale, lam, out_scale, eps, vdim, softcap, chunk):
    """Both maps of a head are rows of one tile, so decoding and prefill each are one launch (and a combine where the context is split) that
    ends with the difference and the head norm. Rows of the tensor-core kernels: 64, 128 or 256 wide; others, and fp32, run the plain kernel.
    Prompts with soft-capped scores (rows of 64 or 128) run on tcgen05."""
    global _LAUNCHES
    T, rows, _ = q.shape
    G, D = kv_cache.shape[2], kv_cache.shape[4]
    out = torch.empty(T, rows // 2, vdim, dtype=q.dtype, device=q.device)
    common = (md.query_start_loc, md.seq_lens, md.block_table, scale)
    if q.dtype == torch.float32 or D not in (64, 128, 256) or rows // G > 64:
        tiles = sum(-(-n * (rows // G) // 16) for n in md.query_lens_cpu)
        _C.diff_attention(q, kv_cache, out, *common, 3, tiles, 1, md.max_query_len, 0, None, None, softcap, chunk, lam, out_scale, eps)
        _LAUNCHES += 1
        return out
    key = ("diff", rows, G, D, chunk)
    plans = md.__dict__.setdefault("_diff_plans", {})
    if key not in plans:
        plans[key] = plan_attention(md.query_lens_cpu, md.seq_lens_cpu, rows, G, D, _sms(q.device), span=attention_span(chunk, 0))
    short, tiles, splits = plans[key]
    if any(0 < n <= short for n in md.query_lens_cpu):
        ws_o = ws_ml = None
        if splits > 1:
            w = workspace(q.device)
            ws_o, ws_ml = (w.attn_static if getattr(md, "static_ws", False) else w.attn)(splits * T * rows * D, splits * T * rows * 2)
        _C.diff_attention(q, kv_cache, out, *common, 1, 0, splits, md.max_query_len, short, ws_o, ws_ml, softcap, chunk, lam, out_scale, eps)
        _LAUNCHES += 2 if splits > 1 else 1
    if tiles and max(md.query_lens_cpu) >= DIFF_PREFILL_MIN_LEN and _C.diff_prefill_tc_sizes(D, softcap):
        tiles = sum(-(-n // 128) for n in md.query_lens_cpu if n > short)
        _C.diff_attention(q, kv_cache, out, *common, 2, tiles, 1, md.max_query_len, short, None, None, softcap, chunk, lam, out_scale, eps)
        _LAUNCHES += 1
    elif tiles:
        _C.diff_attention(q, kv_cache, out, *common, 0, tiles, 1, md.max_query_len, short, None, None, softcap, chunk, lam, out_scale, eps)
        _LAUNCHES += 1
    return out


# ----------------------------------------------------------------------------- ops still served by device-side PyTorch
GDN_CHUNK_MIN_LEN = 64  # sequences with at least this many new tokens take the chunked (tensor-core) kernels


def _gdn_chunk_meta(md, device):
    """Chunk list of this step for the chunked Gated-DeltaNet kernels, built once per step from the host-side query lengths:
    int32 ``[chunk_req | chunk_t0 | long_req | long_chunk0]`` on the device (asynchronous copy from pinned memory)."""
    cached = getattr(md, "_gdn_chunks", None)
    if cached is not None:
        return cached
    qlens = getattr(md, "query_lens_cpu", None)
    meta, nc, nl = None, 0, 0
    if qlens and max(qlens) >= GDN_CHUNK_MIN_LEN and not getattr(md, "is_uniform_decode", False):
        creq, ct0, lreq, lc0 = [], [], [], []
        t = 0
        for r, n in enumerate(qlens):
            if n >= GDN_CHUNK_MIN_LEN:
                lreq.append(r)
                lc0.append(len(creq))
                for c in range(0, n, 64):
                    creq.append(r)
                    ct0.append(t + c)
            t += n
        nc, nl = len(creq), len(lreq)
        host = torch.tensor(creq + ct0 + lreq + lc0, dtype=torch.int32).pin_memory()
        meta = host.to(device, non_blocking=True)
        md._gdn_chunks_host = host  # keep the pinned buffer alive until the copy has run
    md._gdn_chunks = (meta, nc, nl)
    return md._gdn_chunks


def gdn_forward(mixed, b, a, conv_w, A_log, dt_bias, conv_state, ssm_state, md, Hk, Hv, K, V):
    """Conv + gating + gated delta rule. Short sequences (decode, verification) run the recurrent kernel; sequences of at least
    ``GDN_CHUNK_MIN_LEN`` new tokens run the chunked tensor-core kernels. Under speculative verification (``md.gdn_record`` set by
    the runner) the slots are left untouched and the state after every token is recorded for the later commit."""
    global _LAUNCHES
    _LAUNCHES += 3
    rec = getattr(md, "gdn_record", None)
    hi = md.has_initial_state if md.has_initial_state.dtype == torch.int32 else md.has_initial_state.to(torch.int32)
    if rec is None:
        meta, nc, nl = _gdn_chunk_meta(md, mixed.device) if os.environ.get("ONECAT_GDN_PREFILL", "chunked") == "chunked" else (None, 0, 0)
        if nl:
            _LAUNCHES += 2
        return _C.gdn_forward(mixed, b, a, conv_w.to(torch.bfloat16), A_log, dt_bias, conv_state, ssm_state, md.query_start_loc, md.state_slots,
                              hi, Hk, Hv, K, V, True, None, meta, nc, nl, GDN_CHUNK_MIN_LEN)
    q = md.spec_q
    spec = torch.empty(md.num_reqs, q, Hv, K, V, dtype=torch.float32, device=mixed.device)
    prev = conv_state[md.state_slots.long()].clone()
    out = _C.gdn_forward(mixed, b, a, conv_w.to(torch.bfloat16), A_log, dt_bias, conv_state, ssm_state, md.query_start_loc, md.state_slots,
                         hi, Hk, Hv, K, V, False, spec, None, 0, 0, 0)
    rec.append(dict(conv_state=conv_state, ssm_state=ssm_state, spec=spec, prev=prev, mixed=mixed, kw=conv_w.shape[1]))
    return out


def gdn_commit(md, rec: list, n_valid: torch.Tensor) -> None:
    """After verification: every Gated-DeltaNet layer takes the state that follows the last accepted token."""
    global _LAUNCHES
    hi = md.has_initial_state if md.has_initial_state.dtype == torch.int32 else md.has_initial_state.to(torch.int32)
    slots = md.state_slots.long()
    ar = torch.arange(md.num_reqs, device=n_valid.device)
    idx = (n_valid.long() - 1).clamp(min=0)
    qlen = md.query_start_loc[1:] - md.query_start_loc[:-1]
    recorded = qlen <= md.spec_q  # longer sequences (prefill chunks) wrote their slot directly
    rs, ridx = slots[recorded], ar[recorded]
    for e in rec:
        e["ssm_state"][rs] = e["spec"][ridx, idx[recorded].clamp(max=e["spec"].shape[1] - 1)]
        _C.gdn_conv_commit(e["mixed"], e["conv_state"], e["prev"], n_valid.to(torch.int32), md.query_start_loc, md.state_slots, hi, e["kw"])
        _LAUNCHES += 2


def prepare_moe(moe) -> None:
    """Stack the local experts for the grouped GEMM. bf16 experts: ``w13`` → ``[E*2I, H]`` with each expert's gate|up rows
    interleaved in blocks of 16 (SiLU·mul happens in the GEMM epilogue), ``w2`` → ``[E*H, I]``. Block-scaled FP8 and MXFP4 experts
    stay packed: tiles + scale words of the stacked matrices, dequantised inside the GEMM."""
    E, I2 = moe.w13.shape[0], moe.w13.shape[1]
    I = I2 // 2
    H = moe.w2.shape[1]
    if moe.w13.dtype == torch.float32:
        moe.kernel_state = dict(f32=True)   # engines that run in 32 bits: the weights as they are
        return
    if (I2 % 128 or H % 128 or I % 64) and moe.qmethod == "none":
        # sizes that are no multiples of the kernel's tiles: zero rows and columns (a padded gate row gives silu(0) * 0)
        Ip, Hp = -(-I // 64) * 64, -(-H // 128) * 128
        pad = torch.nn.functional.pad
        w13 = pad(moe.w13.data.view(E, 2, I, H), (0, Hp - H, 0, Ip - I)).reshape(E, 2 * Ip, Hp)
        moe.w13 = torch.nn.Parameter(w13, requires_grad=False)
        moe.w2 = torch.nn.Parameter(pad(moe.w2.data, (0, Ip - I, 0, Hp - H)), requires_grad=False)
        I, I2, H = Ip, 2 * Ip, Hp
    if I2 % 128 or H % 128 or I % 64:
        moe.kernel_state = None  # odd shapes of packed experts take the device-side PyTorch path
        return
    perm = interleave_gate_up(I, moe.w13.device)
    q = moe.qmethod
    bn, bk = getattr(moe, "block", None) or (128, 128)
    if q == "fp8" and bk % 64 == 0 and H % bk == 0 and I % bk == 0:
        s13 = moe.w13_scale.float().repeat_interleave(bn, dim=1)[:, :I2][:, perm].reshape(E * I2, -1)
        s2 = moe.w2_scale.float().repeat_interleave(bn, dim=1)[:, :H].reshape(E * H, -1)
        t13, z13, _ = pack_fp8(moe.w13.data.view(torch.uint8)[:, perm].reshape(E * I2, H), s13.contiguous(), bk)
        t2, z2, _ = pack_fp8(moe.w2.data.view(torch.uint8).reshape(E * H, I), s2.contiguous(), bk)
        moe.kernel_state = dict(w13=t13, w2=t2, w13_sz=z13, w2_sz=z2, wkind=2, I2=I2, gk=bk // 64)
    elif q == "mxfp4":
        t13, z13, _ = pack_mxfp4(moe.w13.data[:, perm].reshape(E * I2, H // 2).contiguous(), moe.w13_scale.data[:, perm].reshape(E * I2, -1).contiguous())
        t2, z2, _ = pack_mxfp4(moe.w2.data.reshape(E * H, I // 2).contiguous(), moe.w2_scale.data.reshape(E * H, -1).contiguous())
        moe.kernel_state = dict(w13=t13, w2=t2, w13_sz=z13, w2_sz=z2, wkind=3, I2=I2, gk=1)
    else:
        w13, w2 = moe.dequantized()
        w13s = w13.to(torch.bfloat16)[:, perm, :].reshape(E * I2, H).contiguous()
        w2s = w2.to(torch.bfloat16).reshape(E * H, I).contiguous()
        moe.kernel_state = dict(w13=w13s, w2=w2s, wkind=0)
        if q == "none":  # the stacked copies replace the originals
            moe._dq = None
            moe.w13 = torch.nn.Parameter(w13s.view(E, I2, H), requires_grad=False)
            moe.w2 = torch.nn.Parameter(w2s.view(E, H, I), requires_grad=False)
            moe.kernel_state = dict(w13=moe.w13.view(E * I2, H), w2=moe.w2.view(E * H, I), wkind=0)
            return
    moe._dq = None
    for n in ("w13", "w2", "w13_scale", "w2_scale"):
        if hasattr(moe, n):
            delattr(moe, n)


def route(logits, cfg, bias):
    """Top-k experts and their weights from the router logits (bf16, or fp32 for routers that keep the accumulator's precision)."""
    global _LAUNCHES
    if logits.shape[1] > 512 or cfg.num_experts_per_tok > 16:
        TORCH_STANDINS.add("route")
        if cfg.scoring_func == "sigmoid" or cfg.n_group > 1:
            return ref.grouped_topk(logits, cfg.num_experts_per_tok, cfg.n_group, cfg.topk_group, bias, cfg.scoring_func, cfg.norm_topk_prob,
                                    cfg.routed_scaling_factor)
        return ref.topk_softmax(logits, cfg.num_experts_per_tok, cfg.norm_topk_prob)
    _LAUNCHES += 1
    deepseek = cfg.scoring_func == "sigmoid" or cfg.n_group > 1
    return _C.route(logits if logits.dtype == torch.float32 else logits.to(torch.bfloat16), bias, cfg.num_experts_per_tok,
                    cfg.n_group if deepseek else 1, cfg.topk_group if deepseek else 1,
                    cfg.scoring_func == "sigmoid", cfg.norm_topk_prob, cfg.routed_scaling_factor if deepseek else 1.0)


def fused_moe(moe, x, topk_w, topk_ids):
    global _LAUNCHES
    ks = moe.kernel_state
    if ks is None:
        TORCH_STANDINS.add("fused_moe")
        w13, w2 = moe.dequantized()
        return ref.fused_experts(x, w13, w2, topk_w, topk_ids, moe.e_off)
    ws = workspace(x.device)
    _LAUNCHES += 7
    if ks.get("f32"):
        return _C.fused_moe_f32(x.contiguous(), moe.w13.data, moe.w2.data, topk_w.contiguous().float(), topk_ids.contiguous().to(torch.int32), moe.e_off)
    if x.stride(-1) != 1 or (x.stride(0) * 2) % 16:
        x = x.contiguous()
    return _C.fused_moe(x, ks["w13"], ks["w2"], topk_w.contiguous().float(), topk_ids.contiguous().to(torch.int32), moe.E_local, moe.e_off,
                        ws.splitk, ws.counters, ks.get("wkind", 0), ks.get("w13_sz"), ks.get("w2_sz"), ks.get("I2", 0), ks.get("gk", 1))


# ----------------------------------------------------------------------------- latent attention
MLA_WIDTHS = (64, 128, 192, 256, 384, 512)   # latents the tensor-core kernel has variants for


def mla_padded_sizes(lora: int, rope: int) -> tuple[int, int]:
    """(latent, key part) widths of a cached bf16 row: the next sizes of the tensor-core kernel (zeros in between), or the sizes as they are
    when it has none."""
    lp, rp = next((w for w in MLA_WIDTHS if w >= lora), 0), -(-rope // 16) * 16
    return (lp, rp) if lp and _C.mla_tensor_core_sizes(lp, rp) else (lora, rope)


def mla_prepare(q_latent, kv, q_w, kv_w, eps, positions, cos_sin, cache, slot_mapping, lora, lora_pad, interleaved):
    global _LAUNCHES
    _LAUNCHES += 1
    if q_latent is not None and q_latent.stride(-1) != 1:
        q_latent = q_latent.contiguous()
    return _C.mla_prepare(q_latent, kv if kv.stride(-1) == 1 else kv.contiguous(), None if q_w is None else q_w.to(kv.dtype), kv_w.to(kv.dtype), eps,
                          positions.to(torch.int32), cos_sin, cache, slot_mapping.to(torch.int32), lora, lora_pad, interleaved)


def per_head_matmul(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``x`` ``[T, H, a]`` (strided) times ``w`` ``[H, a, b]`` per head -> contiguous ``[T, H, b]`` (library batched product, written in place)."""
    if x.dtype == torch.float32 and torch.backends.cuda.matmul.allow_tf32:
        raise RuntimeError("fp32 models need torch.backends.cuda.matmul.allow_tf32 = False")
    out = torch.empty(x.shape[0], x.shape[1], w.shape[2], dtype=x.dtype, device=x.device)
    torch.bmm(x.transpose(0, 1), w, out=out.transpose(0, 1))
    return out


def plan_mla_splits(H: int, lora: int, query_lens: list, seq_lens: list, num_sms: int) -> int:
    """KV splits of a latent-attention launch: as many CTAs fit an SM as two key tiles and the queries leave room for."""
    per_sm = max(1, min(4, (227 << 10) // ((16 + 2 * 64) * (lora + 64) * 2 + 6144)))
    return choose_decode_splits(len(query_lens) * -(-max(query_lens) * H // 16), max(seq_lens), num_sms, per_sm)


def mla_decode(q_abs, q_pe, latent_cache, md, scale, lora, cos_sin=None, interleaved=True, fine=False, skip_min_len=0, sinks=None, gate=None):
    """Multi-query attention over the cached latents: ``q_abs`` ``[T, H, lora]``, ``q_pe`` ``[T, H, rope]`` (rotated by the kernel when
    ``cos_sin`` is given). ``fine``: softmax weights in two bf16 terms. ``skip_min_len``: requests with at least that many new tokens are
    left out (their rows of the result hold nothing). ``sinks`` fp32 ``[H]`` join the softmax denominator; ``gate`` ``[T, H]``: logits of a
    per-head output gate."""
    global _LAUNCHES
    T, H, _ = q_abs.shape
    ws_o = ws_ml = None
    splits = 1
    ql, sl = md.query_lens_cpu or [md.max_query_len] * md.num_reqs, md.seq_lens_cpu or [md.max_seq_len]
    if skip_min_len:
        keep = [(q, s) for q, s in zip(ql, sl) if 0 < q < skip_min_len]
        ql, sl = [q for q, _ in keep], [s for _, s in keep]
    if q_abs.dtype == torch.bfloat16 and _C.mla_tensor_core_sizes(lora, latent_cache.shape[-1] - lora):
        static = getattr(md, "static_ws", False)
        plan = getattr(md, "attn_plan", None)
        if static and plan is not None and plan[0][0] == "mla":
            splits = plan[1][2]  # captured decode graph: the split count is part of the graph's key
        else:
            splits = plan_mla_splits(H, lora, ql, sl, _sms(q_abs.device))
        if splits > 1:
            w = workspace(q_abs.device)
            ws_o, ws_ml = (w.attn_static if static else w.attn)(splits * T * H * lora, splits * T * H * 2)
    _LAUNCHES += 2 if splits > 1 else 1
    return _C.mla_decode(q_abs, q_pe, latent_cache, md.query_start_loc, md.seq_lens, md.block_table, scale, max(ql), splits, ws_o, ws_ml, cos_sin,
                         interleaved, fine, skip_min_len, sinks, gate)


MLA_PREFILL_MIN_LEN = 64           # portions of at least this many tokens attend in the expanded form
MLA_PREFILL_BYTES = 4 << 30        # most memory of a step's expanded keys and values; beyond it the absorbed form runs


def mla_prefill_plan(md, H: int, nope: int, rope: int, vd: int, lora_pad: int, device):
    """(metadata, requests, context rows, query tiles, whether shorter portions remain) of the requests that attend in the expanded form in
    this step, or None; built once per step from the host-side lengths."""
    cache = md.__dict__.setdefault("_mla_prefill", {})
    key = (H, nope, rope, vd, lora_pad)
    if key in cache:
        return cache[key]
    ql, sl = getattr(md, "query_lens_cpu", None), getattr(md, "seq_lens_cpu", None)
    out = None
    if ql and sl and max(ql) >= MLA_PREFILL_MIN_LEN and not getattr(md, "is_uniform_decode", False) and _C.mla_prefill_sizes(nope, rope, vd):
        reqs = [r for r, n in enumerate(ql) if n >= MLA_PREFILL_MIN_LEN]
        rows = sum(sl[r] for r in reqs)
        chunks = lambda n: -(-n // 64) * 64
        if rows * (H * (chunks(nope) + chunks(vd)) + chunks(rope) + lora_pad) * 2 <= MLA_PREFILL_BYTES:
            start, at = [], 0
            for r in reqs:
                start.append(at)
                at += sl[r]
            host = torch.tensor(reqs + start, dtype=torch.int32).pin_memory()
            md.__dict__.setdefault("_mla_hosts", []).append(host)   # keep the pinned buffer alive until the copy has run
            out = (host.to(device, non_blocking=True), len(reqs), rows, sum(-(-ql[r] // 128) for r in reqs), any(0 < n < MLA_PREFILL_MIN_LEN for n in ql))
    cache[key] = out
    return out


def mla_prefill(plan, q, latent_cache, md, expand, out, nope, rope, lora_pad, scale, cos_sin, interleaved, fine, sinks=None, gate=None):
    """Causal attention of the planned requests in the expanded form, into their rows of ``out`` ``[T, H, vd]``. ``expand(latents)`` is the
    per-head up-projection ``[rows, H * (keys | values)]`` with both parts padded to 64 columns."""
    global _LAUNCHES
    meta, n, rows, tiles, _ = plan
    _LAUNCHES += 3
    lat, rot, qp = _C.mla_prefill_inputs(q, latent_cache, md.query_start_loc, md.block_table, md.positions, meta, n, rows, nope, lora_pad, cos_sin, interleaved)
    _C.mla_prefill(qp, expand(lat), rot, out, md.query_start_loc, md.seq_lens, meta, n, tiles, nope, rope, scale, fine, sinks, gate)
    return out


# ----------------------------------------------------------------------------- mLSTM
CHUNK_MIN_LEN = 64                 # portions of at least this many tokens take the chunked (tensor-core) kernels
CHUNK_SEGMENT_BYTES = 256 << 20    # what a segment keeps per chunk (measured: smaller ones pay in half-filled waves what they save in traffic)


def _chunk_segments(md, per: int, device):
    """(device tensor, [(offset, chunks, sequences)], whether short portions remain) of this step's list of 64-token chunks, built once per step
    from the host-side query lengths and cut into segments of ``per`` chunks, which bounds the memory of what is kept per chunk."""
    cache = md.__dict__.setdefault("_chunk_segments", {})
    if per in cache:
        return cache[per]
    qlens = getattr(md, "query_lens_cpu", None)
    out = (None, [], True)
    if qlens and max(qlens) >= CHUNK_MIN_LEN and not getattr(md, "is_uniform_decode", False):
        chunks, t = [], 0
        for r, n in enumerate(qlens):
            if n >= CHUNK_MIN_LEN:
                chunks += [(r, t + c) for c in range(0, n, 64)]
            t += n
        flat, segs = [], []
        for a in range(0, len(chunks), per):
            part = chunks[a:a + per]
            reqs, first, count, owner = [], [], [], []
            for j, (r, _) in enumerate(part):
                if not reqs or reqs[-1] != r:
                    reqs.append(r)
                    first.append(j)
                    count.append(0)
                count[-1] += 1
                owner.append(len(reqs) - 1)
            segs.append([len(flat), len(part), len(reqs)])
            flat += [r for r, _ in part] + [t0 for _, t0 in part] + owner + reqs + first + count
        host = torch.tensor(flat, dtype=torch.int32).pin_memory()
        out = (host.to(device, non_blocking=True), segs, any(0 < n < CHUNK_MIN_LEN for n in qlens))
        md.__dict__.setdefault("_chunk_hosts", []).append(host)   # keep the pinned buffer alive until the copy has run
    cache[per] = out
    return out


def mlstm(qkvg, gates, i_bias, f_bias, norm_w, eps, cap, H, D, V, state, md):
    """Short portions (decoding included) run the recurrent kernel, portions of at least ``CHUNK_MIN_LEN`` tokens the chunked ones
    (bf16); both include the head norm and the output gate."""
    global _LAUNCHES
    hi = md.has_initial_state if md.has_initial_state.dtype == torch.int32 else md.has_initial_state.to(torch.int32)
    meta, segs, short = (None, [], True) if qkvg.dtype == torch.float32 or not _C.mlstm_chunkable(D, V) else \
        _chunk_segments(md, max(8, CHUNK_SEGMENT_BYTES // (8 * H * D * V)), qkvg.device)
    _LAUNCHES += 3 * len(segs) + int(short or not segs)
    S, n, m = state
    return _C.mlstm(qkvg, gates, i_bias, f_bias, norm_w, eps, cap, H, D, V, S, n, m, md.query_start_loc, md.state_slots, hi, meta, segs,
                    CHUNK_MIN_LEN, short)


# ----------------------------------------------------------------------------- short convolutions, matrix-state recurrences
def _int32(t):
    return t if t.dtype == torch.int32 else t.to(torch.int32)


def causal_conv(x, weight, bias, state, md, silu=False, residual=False):
    global _LAUNCHES
    _LAUNCHES += 1
    return _C.causal_conv(x, weight, bias, state, md.query_start_loc, md.state_slots, _int32(md.has_initial_state), silu, residual)


def channel_delta(qkv, a, b, A_log, dt_bias, state, md, Hk, H, D, V):
    """Short portions (decoding included) run the recurrent kernel, portions of at least ``CHUNK_MIN_LEN`` tokens the chunked ones (bf16)."""
    global _LAUNCHES
    meta, segs, short = (None, [], True) if qkv.dtype == torch.float32 or not _C.recurrence_chunkable(D, V) else \
        _chunk_segments(md, max(8, CHUNK_SEGMENT_BYTES // (H * _C.delta_chunk_bytes(D, V))), qkv.device)
    _LAUNCHES += 2 * len(segs) + int(short or not segs)
    return _C.recurrence(qkv, a, b, A_log, dt_bias, None, state, md.query_start_loc, md.state_slots, _int32(md.has_initial_state), Hk, H, D, V, 0.0,
                         float("inf"), meta, segs, CHUNK_MIN_LEN, short)


def mamba2(xbc, dt, A_log, dt_bias, D, state, md, H, G, N, V, dt_limit):
    """As ``channel_delta``; the chunked kernel keeps nothing per chunk, so its list is one segment."""
    global _LAUNCHES
    meta, segs, short = (None, [], True) if xbc.dtype == torch.float32 or not _C.recurrence_chunkable(N, V) else _chunk_segments(md, 1 << 30, xbc.device)
    _LAUNCHES += len(segs) + int(short or not segs)
    return _C.recurrence(xbc, None, dt, A_log, dt_bias, D, state, md.query_start_loc, md.state_slots, _int32(md.has_initial_state), G, H, N, V,
                         dt_limit[0], dt_limit[1], meta, segs, CHUNK_MIN_LEN, short)


def gated_norm(x, gate, w, eps, groups, gate_first):
    global _LAUNCHES
    _LAUNCHES += 1
    return _C.gated_norm(x, gate, w, eps, groups, gate_first)


# ----------------------------------------------------------------------------- talking-heads attention
TALK_WS_BYTES = 256 << 20   # partial results of a prompt's tiles that are in memory at a time
TALK_ROWS = 592             # partial rows of single tokens (requests times key splits), four per SM


def talk_row(H: int, G: int, dim: int) -> int:
    """Width of a cached bf16 row: padded for the tensor-core kernels, or as it is where only the plain kernel serves the sizes."""
    return _C.talk_tc_row(H, G, dim) or dim


def talk_workspace(H: int, G: int, D: int, tokens: int) -> tuple[int, int]:
    """Most elements of the partial results and of the sums that decode steps of up to ``tokens`` requests need."""
    rows = max(tokens, TALK_ROWS)
    return rows * H * G * D, rows * H * 2


def talk_prepare(qk, q_gain, eps, temperature, positions, pages, k_scale, slot_mapping, heads, kv_heads, dim):
    global _LAUNCHES
    _LAUNCHES += 1
    coef, every = temperature or (0.0, 0)
    return _C.talk_prepare(qk, q_gain, eps, coef, every, _int32(positions), pages, k_scale, _int32(slot_mapping), heads, kv_heads, dim)


def plan_talk(query_lens: list, seq_lens: list, num_sms: int) -> tuple[int, int]:
    """(key splits of the single tokens, 0 without any; 128-token tiles of the longer portions)."""
    longest = max((s for q, s in zip(query_lens, seq_lens) if q == 1), default=0)
    splits = max(1, min(choose_decode_splits(query_lens.count(1), longest, num_sms, 1), TALK_ROWS // len(query_lens))) if longest else 0
    return splits, sum(-(-q // 128) for q in query_lens if q > 1)


def talk_attention(q, pages, k_scale, md, bias, mix, dim):
    """Talking-heads attention: single tokens and longer portions run tensor-core kernels of their own for the sizes they take; the plain kernel
    serves the rest and fp32."""
    global _LAUNCHES
    T, H, row = q.shape
    G = pages.shape[2]
    out = torch.empty(T, H, dim, dtype=q.dtype, device=q.device)
    args = (q, pages, k_scale, bias, mix, out, md.query_start_loc, md.seq_lens, md.block_table, H, dim)
    if q.dtype != torch.bfloat16 or not _C.talk_tc_row(H, G, dim):
        _LAUNCHES += 1
        _C.talk_plain(*args)
        return out
    plan = md.__dict__.get("_talk_plan")
    if plan is None:
        plan = md.__dict__["_talk_plan"] = plan_talk(md.query_lens_cpu, md.seq_lens_cpu, _sms(q.device))
    splits, tiles = plan
    w = workspace(q.device)
    if splits:
        ws_o, ws_ml = (w.attn_static if getattr(md, "static_ws", False) else w.attn)(splits * md.num_reqs * H * G * row, splits * md.num_reqs * H * 2)
        _C.talk_decode(*args, splits, ws_ml, ws_o)
        _LAUNCHES += 2
    if tiles:
        segment = min(tiles, max(1, TALK_WS_BYTES // (4 * 128 * H * G * row)))
        ws_o, ws_ml = w.attn(segment * 128 * H * G * row, segment * 128 * H * 2)
        _C.talk_prefill(*args, tiles, segment, ws_ml, ws_o)
        _LAUNCHES += 2 * -(-tiles // segment)
    return out


def sigmoid_mul(x, gate):
    global _LAUNCHES
    _LAUNCHES += 1
    return _C.sigmoid_mul(x, gate)


_REJ_STEP = [0]


def rejection_sample(draft_ids, num_draft, target_logits, bonus_ids, md, draft_probs, uniforms, synthetic_rates, gen):
    """Draft probabilities are not used: proposers here emit point-mass (greedy) drafts, for which q(x) = 1."""
    global _LAUNCHES
    _LAUNCHES += 2
    _REJ_STEP[0] += 1
    temp = None if md.all_greedy else md.temperature
    rates = torch.tensor(synthetic_rates, dtype=torch.float32, device=target_logits.device) if synthetic_rates is not None else None
    seed = (gen.initial_seed() if gen is not None else 0) * 1000003 + _REJ_STEP[0]
    return _C.rejection_sample(draft_ids.contiguous(), num_draft, target_logits, bonus_ids, uniforms.contiguous(), temp, rates, seed, not md.all_greedy)

"""Prefill and decode throughput of a design beside the closest models of equal size, and its kernels beside theirs.

``python bench.py --design gabisun|sepirax|lodevik|nalasun`` prints one JSON line per size. Random weights and token ids. Model throughput is device time
of engine steps (CUDA events); kernels are timed alone with the L2 flushed before every launch.

Gabisun: the models share width, heads, head size, window, layer runs, vocabulary and tied embeddings: Starcoder2 (layer norms, ungated
GELU feed-forward of the same width; its norms are PyTorch operations) and Mistral (every step fused; RMS norms, a gated feed-forward of
2/3 the width, so the same number of weights).

Sepirax: beside DeepSeek-V2 (every layer latent attention with the same heads, latents and grouped softmax experts) and Qwen3-Next (Gated-
DeltaNet in the place of the mLSTM layers with the same number of heads and states of 128 x 128, softmax attention in the place of latent
attention, the same experts without groups).

Lodevik: beside Gemma-2 (soft-capped attention with one map of the same number of columns, a window of the chunk's size in every other layer,
full attention in the rest, gated GELU, norms ahead of and behind the sub-blocks) and a dense DeepSeek-V2 (every layer latent attention with
the same heads and latents, gated SiLU).

Nalasun (talking-heads attention, channel delta rule and Mamba-2 in turn): beside Qwen3-Next (Gated-DeltaNet in two of three layers, softmax
attention with the same heads in the third, the same experts and shared expert) and Granite 4 hybrid (Mamba-2 in two of three layers, softmax attention in
the third, the same experts and shared expert). Kernels of the attention layers also beside Gabisun's, whose values are its keys as well."""
from __future__ import annotations

import gc
import json

import torch

SIZES = {
    # width, query heads, kv heads, head size, feed-forward, layers, loop, window, kept tokens, scale
    "w2048": dict(width=2048, heads=16, kv=4, dim=128, ff=8192, layers=12, loop=(2, 6, 2), window=1024, keep=64),
    "w4096": dict(width=4096, heads=32, kv=8, dim=128, ff=16384, layers=8, loop=(2, 4, 2), window=4096, keep=128),
    "w2048d64": dict(width=2048, heads=32, kv=8, dim=64, ff=8192, layers=12, loop=(2, 6, 2), window=1024, keep=64),
}
VOCAB, BIAS_MAX = 32000, 128
PREFILL, DECODE_REQS, DECODE_CTX = 8192, 64, 4096


def gabisun_config(s: dict) -> dict:
    layer = dict(type="attention", mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=s["dim"], vdim=s["dim"], scale=s["dim"] ** -0.5, bias_max=BIAS_MAX,
                 mask=dict(size=s["window"], keep_first=s["keep"])), mlp=dict(kind="dense", ff=s["ff"]))
    return dict(architecture="Gabisun", width=s["width"], vocab=VOCAB, norm=dict(eps=1e-5), layers=[layer] * s["layers"],
                loop=dict(zip(("start", "stop", "times"), s["loop"])))


def like_config(s: dict, arch: str) -> dict:
    a, b, times = s["loop"]
    cfg = dict(architectures=[arch], hidden_size=s["width"], num_hidden_layers=s["layers"] + (times - 1) * (b - a), num_attention_heads=s["heads"],
               num_key_value_heads=s["kv"], head_dim=s["dim"], vocab_size=VOCAB, tie_word_embeddings=True, max_position_embeddings=32768,
               sliding_window=s["window"], rope_theta=10000.0)
    if arch.startswith("Starcoder2"):
        return dict(cfg, intermediate_size=s["ff"], hidden_act="gelu_pytorch_tanh", norm_epsilon=1e-5, use_bias=False)
    return dict(cfg, intermediate_size=s["ff"] * 2 // 3 // 64 * 64, rms_norm_eps=1e-5)


def model_throughput(cfg: dict, steps: int, warmup: int) -> dict:
    """Device time per step of (a) 8192-token prefill steps, (b) decode steps of 64 requests at a context of about 4096 tokens."""
    from onecat_vllm.config import EngineArgs
    from onecat_vllm.engine.llm_engine import LLMEngine
    from onecat_vllm.sampling_params import SamplingParams
    eng = LLMEngine.from_engine_args(EngineArgs(hf_config=cfg, dtype="bfloat16", device="cuda", max_model_len=2 * PREFILL, max_num_seqs=DECODE_REQS,
                                                max_num_batched_tokens=PREFILL, enable_prefix_caching=False, async_scheduling=False, disable_log_stats=False,
                                                kv_cache_memory_bytes=24 << 30))
    g, n = torch.Generator().manual_seed(0), [0]

    def add(length, out):
        n[0] += 1
        eng.add_request(f"r{n[0]}", torch.randint(0, VOCAB, (length,), generator=g).tolist(),
                        SamplingParams(temperature=0.0, max_tokens=out, ignore_eos=True, detokenize=False))

    def step():
        eng.step()
        st = eng.last_scheduler_stats
        return st.step_device_ms, st.num_scheduled_tokens

    ms = []
    for i in range(warmup + max(4, steps // 4)):
        add(PREFILL, 1)
        t, tok = step()
        assert tok == PREFILL
        if i >= warmup:
            ms.append(t)
    out = dict(prefill_ms=sorted(ms)[len(ms) // 2])
    out["prefill_tokens_per_s"] = PREFILL / out["prefill_ms"] * 1e3
    for _ in range(DECODE_REQS):
        add(DECODE_CTX, warmup + steps + 80)
    ms = []
    while len(ms) < warmup + steps:
        t, tok = step()
        if tok == DECODE_REQS:
            ms.append(t)
    ms = sorted(ms[warmup:])
    out["decode_ms"] = ms[len(ms) // 2]
    out["decode_tokens_per_s"] = DECODE_REQS / out["decode_ms"] * 1e3
    eng.shutdown()
    del eng
    gc.collect()
    torch.cuda.empty_cache()
    return out


def _meta(R, q, S):
    from onecat_vllm.worker.attn_metadata import AttentionMetadata
    nb = -(-S // 16)
    bt = (torch.randperm(R * nb, device="cuda").to(torch.int32) + 1).view(R, nb)
    return AttentionMetadata(R, R * q, torch.arange(R + 1, device="cuda", dtype=torch.int32) * q, torch.full((R,), S, device="cuda", dtype=torch.int32), bt,
                             None, None, q, S, query_lens_cpu=[q] * R, seq_lens_cpu=[S] * R), R * nb + 1


def kernel_rows(s: dict, iters: int) -> list[dict]:
    """Each kernel of the design beside the like kernel of the dense models, as fractions of the measured peaks."""
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops.microbench import _peaks, timeit
    pk, rows = _peaks(), []
    W, H, G, D, win, keep = s["width"], s["heads"], s["kv"], s["dim"], s["window"], s["keep"]

    def row(kernel, case, who, fn, flops=0.0, nbytes=0.0):
        ms = timeit(fn, iters)
        t = max(flops / pk["bf16_tflops"] / 1e9, nbytes / pk["hbm_gbs"] / 1e6)
        rows.append(dict(kernel=kernel, case=case, model=who, us=ms * 1e3, roofline_us=t * 1e3, frac_of_roofline=t / ms))

    sinks, table = torch.randn(H, device="cuda"), torch.randn(H, BIAS_MAX + 1, device="cuda")
    for case, R, q, S in (("prefill", 1, PREFILL, PREFILL), ("decode", DECODE_REQS, 1, DECODE_CTX)):
        md, nblk = _meta(R, q, S)
        x = (torch.randn(R * q, H * D + G * D + H, device="cuda") * 0.5).bfloat16()
        qq, gate = x[:, : H * D].view(-1, H, D), x[:, (H + G) * D:]
        pairs = sum(min(i + 1, win) + max(0, min(keep, i + 1 - win)) for i in range(S - q, S)) * R
        keys = min(S, win + keep) * R if q == 1 else S * R
        for who, tensors, kw in (("gabisun", 1, dict(keep=keep, bias_table=table, gate=gate, sinks=sinks)), ("window+sinks", 2, dict(sinks=sinks))):
            cache = (torch.randn(nblk, tensors, G, 16, D, device="cuda") * 0.5).bfloat16()
            md.attn_plan = None
            out = torch.empty(R * q, H, D, dtype=torch.bfloat16, device="cuda")
            row("attention", case, who, lambda: K.paged_attention(qq, cache, md, D ** -0.5, out=out, window=win, **kw), flops=4.0 * H * D * pairs,
                nbytes=2.0 * (keys * tensors * G * D + 2 * R * q * H * D))
            del cache
    for T in (PREFILL, DECODE_REQS):
        b = lambda *sh: torch.randn(*sh, device="cuda").bfloat16()
        part, x32, w, res = b(T, W), torch.randn(T, W, device="cuda"), b(W), b(T, W)
        norm = (2, w, w, 1e-5, False)
        row("norm", T, "gabisun join", lambda: K.stream_join(part, x32, norm, w, norm, torch.bfloat16), nbytes=12.0 * T * W)
        row("norm", T, "add + rms norm", lambda: K.rms_norm(part, w, 1e-5, res, False), nbytes=8.0 * T * W)
        slot = torch.arange(T, device="cuda", dtype=torch.int32)
        kk = b(T, (H + 2 * G) * D)
        ksl = kk[:, H * D: (H + G) * D].view(T, G, D)
        c1, c2 = b(T // 16 + 1, 1, G, 16, D), b(T // 16 + 1, 2, G, 16, D)
        row("cache insert", T, "gabisun", lambda: K.kv_insert(ksl, c1, slot), nbytes=4.0 * T * G * D)
        cs = torch.ones(T, D, device="cuda")
        row("cache insert", T, "rope + insert", lambda: K.rope_and_cache(kk[:, : H * D].view(T, H, D), ksl, kk[:, (H + G) * D:].view(T, G, D), slot, cs, c2, slot, D,
                                                                       None, None, 1e-5, False), nbytes=4.0 * T * (H + 2 * G) * D)

        def gemm(name, who, N, Kd, **kw):
            wt, xx = (torch.randn(N, Kd, device="cuda") * 0.02).bfloat16(), b(T, Kd)
            out = torch.empty(T, -(-N // 8) * 8, dtype=kw.get("out_dtype", torch.bfloat16), device="cuda")[:, :N]
            epi = kw.get("epi", K.EPI_STORE)
            row(f"gemm {name}", T, who, lambda: K._gemm(xx, wt, None, None, out, None, N, N, N // 2 if epi == K.EPI_SILU_MUL else N, 0, epi, 1),
                flops=2.0 * T * N * Kd, nbytes=2.0 * (N * Kd + T * Kd) + out.element_size() * T * N)
        gemm("projections", "gabisun q|k|g", H * D + G * D + H, W)
        gemm("projections", "q|k|v", (H + 2 * G) * D, W)
        gemm("up", "gabisun, GELU epilogue", s["ff"], W, epi=K.EPI_GELU_TANH)
        gemm("up", "gate|up, SiLU epilogue", 2 * (s["ff"] * 2 // 3 // 64 * 64), W, epi=K.EPI_SILU_MUL)
        gemm("loop entry", "gabisun, fp32 output", W, 2 * W, out_dtype=torch.float32)
        gemm("loop entry", "bf16 output", W, 2 * W)
    gemm("logits", "gabisun, fp32 output", VOCAB, W, out_dtype=torch.float32)
    gemm("logits", "bf16 output", VOCAB, W)
    return rows


SEPIRAX_SIZES = {
    # width, layers (mLSTM and latent attention in turn), heads of both, latent attention (dim, rot, vdim, kv rank, q rank), state (dim, vdim), experts
    "w2048": dict(width=2048, layers=12, heads=16, dim=128, rot=64, vdim=128, kv=512, q=768, sdim=128, svdim=128, experts=64, top=6, groups=8, keep=3, ff=512),
    "w4096": dict(width=4096, layers=8, heads=32, dim=128, rot=64, vdim=128, kv=512, q=1536, sdim=128, svdim=128, experts=32, top=4, groups=4, keep=2, ff=1024),
    "w2048s": dict(width=2048, layers=12, heads=32, dim=64, rot=32, vdim=64, kv=256, q=512, sdim=64, svdim=64, experts=16, top=4, groups=4, keep=2, ff=1024),
}


def sepirax_config(s: dict) -> dict:
    mlp = dict(kind="moe", expert=dict(ff=s["ff"]), router=dict(experts=s["experts"], top=s["top"], groups=dict(count=s["groups"], keep=s["keep"])))
    mem = dict(type="mlstm", mlp=mlp, mixer=dict(heads=s["heads"], dim=s["sdim"], vdim=s["svdim"], gate_cap=15.0))
    att = dict(type="latent_attention", mlp=mlp, mixer=dict(heads=s["heads"], dim=s["dim"], rot_dim=s["rot"], vdim=s["vdim"], kv_rank=s["kv"], q_rank=s["q"],
               scale=(s["dim"] + s["rot"]) ** -0.5, rot=dict(base=10000.0, dims=s["rot"], scaling=dict(factor=4.0, fast=32.0, slow=1.0, original=4096))))
    return dict(architecture="Sepirax", width=s["width"], vocab=VOCAB, norm=dict(eps=1e-5), residual_mult=0.5, logit_softcap=30.0,
                embedding=dict(scale=s["width"] ** 0.5), layers=[mem, att] * (s["layers"] // 2))


def sepirax_like(s: dict, arch: str) -> dict:
    cfg = dict(architectures=[arch], hidden_size=s["width"], num_hidden_layers=s["layers"], num_attention_heads=s["heads"], vocab_size=VOCAB,
               max_position_embeddings=32768, rope_theta=10000.0, rms_norm_eps=1e-5, tie_word_embeddings=False, intermediate_size=s["ff"],
               moe_intermediate_size=s["ff"], num_experts_per_tok=s["top"], norm_topk_prob=True)
    if arch.startswith("Deepseek"):
        return dict(cfg, num_key_value_heads=s["heads"], q_lora_rank=s["q"], kv_lora_rank=s["kv"], qk_nope_head_dim=s["dim"], qk_rope_head_dim=s["rot"],
                    v_head_dim=s["vdim"], n_routed_experts=s["experts"], n_shared_experts=0, n_group=s["groups"], topk_group=s["keep"], scoring_func="softmax",
                    first_k_dense_replace=0, routed_scaling_factor=1.0)
    return dict(cfg, num_key_value_heads=max(s["heads"] // 4, 1), head_dim=128, num_experts=s["experts"], shared_expert_intermediate_size=0,
                linear_num_key_heads=s["heads"], linear_num_value_heads=s["heads"], linear_key_head_dim=128, linear_value_head_dim=128,
                linear_conv_kernel_dim=4, full_attention_interval=2, attn_output_gate=True, partial_rotary_factor=0.25)


def sepirax_kernels(s: dict, iters: int) -> list[dict]:
    """Each kernel of the design beside the like kernel of the closest models. Bytes and FLOPs are the algorithm's: what a kernel must read
    and write once, and the products of latent attention in the form that needs fewest of them for its case."""
    from types import SimpleNamespace
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops.microbench import _peaks, timeit
    pk, rows = _peaks(), []
    W, H, L, R, E, top = s["width"], s["heads"], s["kv"], s["rot"], s["experts"], s["top"]
    b = lambda *sh: torch.randn(*sh, device="cuda").bfloat16()
    f32 = lambda *sh: torch.randn(*sh, device="cuda")

    def row(kernel, case, who, fn, flops=0.0, nbytes=0.0):
        ms = timeit(fn, iters)
        t = max(flops / pk["bf16_tflops"] / 1e9, nbytes / pk["hbm_gbs"] / 1e6)
        rows.append(dict(kernel=kernel, case=case, model=who, us=ms * 1e3, roofline_us=t * 1e3, frac_of_roofline=t / ms))

    lp, rp = K.mla_padded_sizes(L, R)
    table = f32(2 * PREFILL, R)
    for case, n, q, S in (("prefill", 1, PREFILL, PREFILL), ("decode", DECODE_REQS, 1, DECODE_CTX)):
        md, nblk = _meta(n, q, S)
        cache, T = b(nblk, 16, lp + rp) * 0.3, n * q
        cache[..., L:lp] = 0
        cache[..., lp + R:] = 0
        pairs = n * sum(range(S - q + 1, S + 1))
        q_abs, q_pe = b(T, H, lp), b(T, H, R)
        if case == "decode":
            fl, by = 2.0 * H * pairs * (2 * L + R), 2.0 * (n * S * (L + R) + T * H * (2 * L + R))
        else:
            fl, by = 2.0 * H * pairs * (s["dim"] + R + s["vdim"]), 2.0 * (S * (L + R) + T * H * (s["dim"] + R + s["vdim"]))
        if case == "prefill":
            # what the engine runs for prompts: latents gathered and expanded, then tcgen05 attention (deepseek: the same with plain weights)
            wkv = b(H * (-(-s["dim"] // 64) * 64 + -(-s["vdim"] // 64) * 64), lp) * 0.05
            md.positions = torch.arange(S, device="cuda", dtype=torch.int32)
            plan = K.mla_prefill_plan(md, H, s["dim"], R, s["vdim"], lp, torch.device("cuda"))
            qq, out = b(T, H, s["dim"] + R), b(T, H, s["vdim"])
            for who, inter, fine in (("sepirax, two-term weights", False, True), ("deepseek", True, False)):
                row("latent attention", case, who, lambda: K.mla_prefill(plan, qq, cache, md, lambda x: K.gemm_bf16(x, wkv), out, s["dim"], R, lp, 0.1, table, inter, fine), fl, by)
            continue
        for who, rest in (("sepirax (rotates q, two-term weights)", (table, False, True)), ("deepseek", (table, True, False))):
            row("latent attention", case, who, lambda: K.mla_decode(q_abs, q_pe, cache, md, 0.1, lp, *rest), fl, by)
        del cache
    for case, n, q in (("prefill", 1, PREFILL), ("decode", DECODE_REQS, 1)):
        T = n * q
        md, _ = _meta(n, q, q)
        md.state_slots = torch.arange(n, device="cuda", dtype=torch.int32)
        md.has_initial_state = torch.ones(n, device="cuda", dtype=torch.int32)
        md.is_uniform_decode = case == "decode"
        for D, V in {(s["sdim"], s["svdim"]), (128, 128)}:
            st = (f32(n, H, D, V), f32(n, H, D), f32(n, H))
            x, g, bi, nw = b(T, 2 * H * (D + V)), f32(T, 2 * H), f32(H), b(H * V)
            cost = lambda D, V: (4.0 * T * H * (D * V + 32 * (D + V)), 2.0 * T * H * (2 * D + 3 * V) + 8.0 * n * H * D * V)
            row("recurrence", case, f"sepirax mLSTM {D}x{V}, head norm and gate included", lambda: K.mlstm(x, g, bi, bi, nw, 1e-5, 15.0, H, D, V, st, md), *cost(D, V))
        D = V = 128
        conv, st = b(n, 3 * H * D, 3), f32(n, H, D, V)
        x, a, cw, al, z, nw = b(T, 3 * H * D), b(T, H), b(3 * H * D, 4), f32(H), b(T, H * V), b(V)
        row("recurrence", case, "qwen3-next Gated-DeltaNet 128x128 with convolution, head norm and gate", lambda: K.rms_norm_gated(
            K.gdn_forward(x, a, a, cw, al, al, conv, st, md, H, H, D, V).reshape(T, H * V), z, nw, 1e-5, H), *cost(D, V))
    for T in (PREFILL, DECODE_REQS):
        part, x32, w, res, al = b(T, W), f32(T, W), b(W), b(T, W), b(1)
        row("norm", T, "sepirax join", lambda: K.stream_join(part, x32, None, None, (3, w, w, 0.0, False, al), torch.bfloat16, mul=0.5), nbytes=12.0 * T * W)
        row("norm", T, "add + rms norm", lambda: K.rms_norm(part, w, 1e-5, res, False), nbytes=8.0 * T * W)
        slot = torch.arange(T, device="cuda", dtype=torch.int32)
        down = b(T, s["q"] + L + R + H * s["vdim"])
        cache, wq, wk = b(T // 16 + 1, 16, lp + rp), b(s["q"]), b(L)
        row("latent norms + rope + insert", T, "sepirax", lambda: K.mla_prepare(down[:, : s["q"]], down[:, s["q"]: s["q"] + L + R], wq, wk, 1e-5, slot, table, cache, slot, L, lp,
                                                                               False), nbytes=4.0 * T * (s["q"] + L + R))
        G = max(H // 4, 1)
        kk, c2, cs = b(T, (H + 2 * G) * 128), b(T // 16 + 1, 2, G, 16, 128), torch.ones(T, 128, device="cuda")
        row("latent norms + rope + insert", T, "rope + insert (qwen3-next)", lambda: K.rope_and_cache(
            kk[:, : H * 128].view(T, H, 128), kk[:, H * 128: (H + G) * 128].view(T, G, 128), kk[:, (H + G) * 128:].view(T, G, 128), slot, cs, c2, slot, 128, None, None,
            1e-5, False), nbytes=4.0 * T * (H + 2 * G) * 128)
        o, gate = b(T, H * s["vdim"]), down[:, s["q"] + L + R:]
        row("output gate", T, "sepirax", lambda: K.sigmoid_mul(o, gate), nbytes=6.0 * T * H * s["vdim"])
        row("output gate", T, "qwen3-next (PyTorch)", lambda: o * torch.sigmoid(gate.float()).to(o.dtype), nbytes=6.0 * T * H * s["vdim"])
        rc = SimpleNamespace(num_experts_per_tok=top, n_group=s["groups"], topk_group=s["keep"], scoring_func="softmax", norm_topk_prob=True, routed_scaling_factor=1.0)
        z = f32(T, E)
        zb = z.bfloat16()
        row("router", T, "sepirax (fp32 logits)", lambda: K.route(z, rc, None), nbytes=T * (4.0 * E + 8.0 * top))
        row("router", T, "deepseek (bf16 logits)", lambda: K.route(zb, rc, None), nbytes=T * (2.0 * E + 8.0 * top))

        def gemm(name, who, N, Kd, **kw):
            wt, xx = (torch.randn(N, Kd, device="cuda") * 0.02).bfloat16(), b(T, Kd)
            out = torch.empty(T, -(-N // 8) * 8, dtype=kw.get("out_dtype", torch.bfloat16), device="cuda")[:, :N]
            row(f"gemm {name}", T, who, lambda: K._gemm(xx, wt, None, None, out, None, N, N, N, 0, K.EPI_STORE, 1), flops=2.0 * T * N * Kd,
                nbytes=2.0 * (N * Kd + T * Kd) + out.element_size() * T * N)
        gemm("latent projections", "sepirax dq|dkv|gate", s["q"] + L + R + H * s["vdim"], W)
        gemm("latent projections", "deepseek q_a", s["q"], W)
        gemm("mixer input", "sepirax q|k|v|gate", 2 * H * (s["sdim"] + s["svdim"]), W)
        gemm("mixer input", "qwen3-next q|k|v|z", 4 * H * 128, W)
        gemm("gates", "sepirax input|forget, fp32 output", 2 * H, W, out_dtype=torch.float32)
        gemm("gates", "qwen3-next b|a", 2 * H, W)
        gemm("router logits", "sepirax, fp32 output", E, W, out_dtype=torch.float32)
        gemm("router logits", "deepseek", E, W)
    return rows


LODEVIK_SIZES = {
    # width, layers (differential and latent attention in turn), heads of both, differential attention (kv heads, dim, vdim, rot, chunk), latent
    # attention (dim, rot, vdim, kv rank), feed-forward
    "w2048": dict(width=2048, layers=12, heads=16, kv=4, dim=64, vdim=128, rot=32, chunk=1024, ldim=128, lrot=64, lvdim=128, lora=512, ff=6144),
    "w4096": dict(width=4096, layers=8, heads=32, kv=8, dim=64, vdim=128, rot=64, chunk=4096, ldim=128, lrot=64, lvdim=128, lora=512, ff=12288),
    "w2048s": dict(width=2048, layers=12, heads=32, kv=8, dim=32, vdim=64, rot=16, chunk=512, ldim=64, lrot=32, lvdim=64, lora=256, ff=6144),
}


def lodevik_config(s: dict) -> dict:
    mlp = dict(kind="dense", ff=s["ff"])
    dif = dict(type="attention", mlp=mlp, mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=s["dim"], vdim=s["vdim"], diff=0.4, scale=s["dim"] ** -0.5, softcap=30.0,
               rot=dict(base=10000.0, dims=s["rot"]), mask=dict(size=s["chunk"])))
    lat = dict(type="latent_attention", mlp=mlp, mixer=dict(heads=s["heads"], dim=s["ldim"], rot_dim=s["lrot"], vdim=s["lvdim"], kv_rank=s["lora"],
               scale=(s["ldim"] + s["lrot"]) ** -0.5, rot=dict(base=500000.0, dims=s["lrot"])))
    return dict(architecture="Lodevik", width=s["width"], vocab=VOCAB, norm=dict(eps=1e-5), logit_scale=0.5, layers=[dif, lat] * (s["layers"] // 2),
                embedding=dict(scale=s["width"] ** 0.5, bigram=dict(buckets=65521, mul_prev=7919, mul_cur=104729)))


def lodevik_like(s: dict, arch: str) -> dict:
    cfg = dict(architectures=[arch], hidden_size=s["width"], num_hidden_layers=s["layers"], num_attention_heads=s["heads"], vocab_size=VOCAB,
               max_position_embeddings=32768, rope_theta=10000.0, rms_norm_eps=1e-5, tie_word_embeddings=True, intermediate_size=s["ff"])
    if arch.startswith("Deepseek"):
        return dict(cfg, num_key_value_heads=s["heads"], kv_lora_rank=s["lora"], qk_nope_head_dim=s["ldim"], qk_rope_head_dim=s["lrot"], v_head_dim=s["lvdim"])
    return dict(cfg, num_key_value_heads=s["kv"], head_dim=2 * s["dim"], query_pre_attn_scalar=2 * s["dim"], attn_logit_softcapping=30.0,
                final_logit_softcapping=None, hidden_activation="gelu_pytorch_tanh", sliding_window=s["chunk"],
                layer_types=["sliding_attention", "full_attention"] * (s["layers"] // 2))


def lodevik_kernels(s: dict, iters: int) -> list[dict]:
    """Each kernel of the design beside the like kernel of the closest models. Bytes and FLOPs are the algorithm's: visible pairs of queries and
    keys, what a kernel must read and write once, and the products of latent attention in the form that needs fewest of them for its case."""
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops.microbench import _peaks, timeit
    pk, rows = _peaks(), []
    W, H, G, D, V, c, L, R = s["width"], s["heads"], s["kv"], s["dim"], s["vdim"], s["chunk"], s["lora"], s["lrot"]
    b = lambda *sh: torch.randn(*sh, device="cuda").bfloat16()
    f32 = lambda *sh: torch.randn(*sh, device="cuda")

    def row(kernel, case, who, fn, flops=0.0, nbytes=0.0):
        ms = timeit(fn, iters)
        t = max(flops / pk["bf16_tflops"] / 1e9, nbytes / pk["hbm_gbs"] / 1e6)
        rows.append(dict(kernel=kernel, case=case, model=who, us=ms * 1e3, roofline_us=t * 1e3, frac_of_roofline=t / ms))

    lam, sink, wide = torch.full((1,), 0.5, device="cuda"), f32(H), 2 * D
    for case, n, q, S in (("prefill", 1, PREFILL, PREFILL), ("decode", DECODE_REQS, 1, DECODE_CTX)):
        T = n * q
        md, nblk = _meta(n, q, S)
        cache = b(nblk, 2, G, 16, wide) * 0.5
        near = lambda seen: (n * sum(seen(i) for i in range(S - q, S)), n * (seen(S - 1) if q == 1 else S))
        qq, x, out = b(T, 2 * H, D), b(T, H, wide), torch.empty(T, H, wide, dtype=torch.bfloat16, device="cuda")
        pairs, keys = near(lambda i: i % c + 1)
        row("attention", case, "lodevik, chunks", lambda: K.diff_attention(qq, cache, md, D ** -0.5, lam, 0.6, 1e-5, V, 30.0, c), 4.0 * H * (D + V) * pairs,
            2.0 * (keys * G * (wide + V) + T * H * (wide + V)))
        pairs, keys = near(lambda i: min(i + 1, c))
        row("attention", case, "gemma-2, window and soft cap", lambda: K.paged_attention(x, cache, md, wide ** -0.5, out=out, window=c, softcap=30.0),
            4.0 * H * wide * pairs, 2.0 * (keys * G * 2 * wide + 2 * T * H * wide))
        pairs, keys = near(lambda i: i + 1)
        md.attn_plan = None
        row("attention", case, "gemma-2, full with soft cap", lambda: K.paged_attention(x, cache, md, wide ** -0.5, out=out, softcap=30.0),
            4.0 * H * wide * pairs, 2.0 * (keys * G * 2 * wide + 2 * T * H * wide))
        del cache
    lp, rp = K.mla_padded_sizes(L, R)
    table = f32(2 * PREFILL, R)
    for case, n, q, S in (("prefill", 1, PREFILL, PREFILL), ("decode", DECODE_REQS, 1, DECODE_CTX)):
        md, nblk = _meta(n, q, S)
        cache, T, pairs, gate = b(nblk, 16, lp + rp) * 0.3, n * q, n * sum(range(S - q + 1, S + 1)), b(n * q, H)
        if case == "prefill":
            wkv = b(H * (-(-s["ldim"] // 64) * 64 + -(-s["lvdim"] // 64) * 64), lp) * 0.05
            md.positions = torch.arange(S, device="cuda", dtype=torch.int32)
            plan = K.mla_prefill_plan(md, H, s["ldim"], R, s["lvdim"], lp, torch.device("cuda"))
            qq, out = b(T, H, s["ldim"] + R), b(T, H, s["lvdim"])
            fl, by = 2.0 * H * pairs * (s["ldim"] + R + s["lvdim"]), 2.0 * (S * (L + R) + T * H * (s["ldim"] + R + s["lvdim"]))
            for who, rest in (("lodevik, two-term weights, sink and gate", (True, sink, gate)), ("deepseek", (False, None, None))):
                row("latent attention", case, who, lambda: K.mla_prefill(plan, qq, cache, md, lambda x: K.gemm_bf16(x, wkv), out, s["ldim"], R, lp, 0.1, table,
                                                                         True, *rest), fl, by)
            continue
        q_abs, q_pe = b(T, H, lp), b(T, H, R)
        fl, by = 2.0 * H * pairs * (2 * L + R), 2.0 * (n * S * (L + R) + T * H * (2 * L + R))
        for who, rest in (("lodevik, two-term weights, sink and gate", (True, 0, sink, gate)), ("deepseek", (False,))):
            row("latent attention", case, who, lambda: K.mla_decode(q_abs, q_pe, cache, md, 0.1, lp, table, True, *rest), fl, by)
        del cache
    for T in (PREFILL, DECODE_REQS):
        part, x32, w, res, y = b(T, W), f32(T, W), b(W), b(T, W), b(T, W)
        row("norm", T, "lodevik join", lambda: K.stream_join(part, x32, (1, w, None, 1e-5, False), w, None, torch.bfloat16, copy_out=y), nbytes=12.0 * T * W)
        row("norm", T, "add + rms norm", lambda: K.rms_norm(part, w, 1e-5, res, False), nbytes=8.0 * T * W)
        ids, prev = (torch.randint(0, VOCAB, (T,), device="cuda", dtype=torch.int32) for _ in range(2))
        emb, big = b(VOCAB, W), b(65522, W)
        row("embedding", T, "lodevik, token and bigram rows", lambda: K.embed_stream(ids, emb, 3.0, prev, big, (7919, 104729), torch.bfloat16), nbytes=10.0 * T * W)
        row("embedding", T, "gemma-2 (PyTorch)", lambda: torch.nn.functional.embedding(ids, emb) * 3.0, nbytes=4.0 * T * W)
        slot = torch.arange(T, device="cuda", dtype=torch.int32)
        kk, cc, cs, nw = b(T, H * wide + G * (wide + V)), b(T // 16 + 1, 2, G, 16, wide), torch.ones(T, s["rot"], device="cuda"), b(D)
        row("norms + rope + insert", T, "lodevik", lambda: K.diff_prepare(kk, nw, nw, 1e-5, slot, cs, cc, slot, H, G, D, V, True), nbytes=4.0 * T * (H * wide + G * (wide + V)))
        k2, cs2, nw2 = b(T, (H + 2 * G) * wide), torch.ones(T, wide, device="cuda"), b(wide)
        row("norms + rope + insert", T, "qwen3", lambda: K.rope_and_cache(k2[:, : H * wide].view(T, H, wide), k2[:, H * wide: (H + G) * wide].view(T, G, wide),
            k2[:, (H + G) * wide:].view(T, G, wide), slot, cs2, cc, slot, wide, nw2, nw2, 1e-5, False), nbytes=4.0 * T * (H + 2 * G) * wide)
        n_in = H * (s["ldim"] + R) + L + R + H
        down, lc, wk = b(T, -(-n_in // 8) * 8), b(T // 16 + 1, 16, lp + rp), b(L)
        row("latent norm + rope + insert", T, "lodevik and deepseek", lambda: K.mla_prepare(None, down[:, H * (s["ldim"] + R): n_in - H], None, wk, 1e-5, slot, table, lc,
                                                                                             slot, L, lp, True), nbytes=4.0 * T * (L + R))

        def gemm(name, who, N, Kd, **kw):
            wt, xx = (torch.randn(N, Kd, device="cuda") * 0.02).bfloat16(), b(T, Kd)
            epi = kw.get("epi", K.EPI_STORE)
            no = N if epi == K.EPI_STORE else N // 2
            out = torch.empty(T, -(-no // 8) * 8, dtype=kw.get("out_dtype", torch.bfloat16), device="cuda")[:, :no]
            row(f"gemm {name}", T, who, lambda: K._gemm(xx, wt, None, None, out, None, N, N, no, 0, epi, 1), flops=2.0 * T * N * Kd,
                nbytes=2.0 * (N * Kd + T * Kd) + out.element_size() * T * no)
        gemm("projections", "lodevik q|k|v", H * wide + G * (wide + V), W)
        gemm("projections", "lodevik latent q|dkv|gate", n_in, W)
        gemm("projections", "deepseek q", H * (s["ldim"] + R), W)
        gemm("gate|up", "lodevik, GELU epilogue", 2 * s["ff"], W, epi=K.EPI_GELU_MUL)
        gemm("gate|up", "SiLU epilogue", 2 * s["ff"], W, epi=K.EPI_SILU_MUL)
    gemm("logits", "lodevik, fp32 output", VOCAB, W, out_dtype=torch.float32)
    gemm("logits", "bf16 output", VOCAB, W)
    return rows


NALASUN_SIZES = {
    # width, layers (attention, channel delta, Mamba-2 in turn), attention (heads, kv heads, dim), delta rule (heads, dim), Mamba-2 (heads, vdim, state,
    # groups), experts (count, chosen, width, shared width)
    "w2048": dict(width=2048, layers=12, heads=16, kv=4, dim=128, dheads=16, ddim=128, mheads=64, mdim=64, state=128, groups=1, experts=64, top=6, ff=512, shared=1024),
    "w4096": dict(width=4096, layers=9, heads=32, kv=8, dim=128, dheads=32, ddim=128, mheads=128, mdim=64, state=128, groups=8, experts=64, top=4, ff=1024, shared=2048),
    "w2048s": dict(width=2048, layers=12, heads=32, kv=8, dim=64, dheads=32, ddim=64, mheads=32, mdim=64, state=64, groups=2, experts=64, top=6, ff=512, shared=1024),
}


def nalasun_config(s: dict) -> dict:
    mlp = dict(kind="moe", expert=dict(ff=s["ff"]), shared=dict(ff=s["shared"]), router=dict(experts=s["experts"], top=s["top"], scale=2.0))
    att = dict(type="attention", mlp=mlp, mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=s["dim"], vdim=s["dim"], scale=s["dim"] ** -0.5, q_temp=dict(coef=0.1, every=4096)))
    dlt = dict(type="channel_delta", mlp=mlp, mixer=dict(heads=s["dheads"], kv_heads=s["dheads"], dim=s["ddim"], vdim=s["ddim"], conv=4))
    ssm = dict(type="mamba2", mlp=mlp, mixer=dict(heads=s["mheads"], vdim=s["mdim"], state=s["state"], groups=s["groups"], norm_groups=s["groups"], conv=4))
    return dict(architecture="Nalasun", width=s["width"], vocab=VOCAB, max_positions=2 * PREFILL, norm=dict(eps=1e-5), canon=dict(taps=4),
                layers=[att, dlt, ssm] * (s["layers"] // 3))


def nalasun_like(s: dict, arch: str) -> dict:
    cfg = dict(architectures=[arch], hidden_size=s["width"], num_hidden_layers=s["layers"], num_attention_heads=s["heads"], num_key_value_heads=s["kv"],
               head_dim=s["dim"], vocab_size=VOCAB, max_position_embeddings=32768, rope_theta=10000.0, rms_norm_eps=1e-5, tie_word_embeddings=True,
               num_experts_per_tok=s["top"])
    if arch.startswith("Granite"):
        return dict(cfg, layer_types=["attention", "mamba", "mamba"] * (s["layers"] // 3), mamba_n_heads=s["mheads"], mamba_d_head=s["mdim"], mamba_d_state=s["state"],
                    mamba_n_groups=s["groups"], mamba_d_conv=4, mamba_expand=s["mheads"] * s["mdim"] / s["width"], intermediate_size=s["ff"],
                    shared_intermediate_size=s["shared"], num_local_experts=s["experts"], attention_multiplier=s["dim"] ** -0.5, embedding_multiplier=1.0,
                    residual_multiplier=1.0, logits_scaling=1.0, position_embedding_type="nope")
    return dict(cfg, intermediate_size=s["ff"], moe_intermediate_size=s["ff"], norm_topk_prob=True, num_experts=s["experts"],
                shared_expert_intermediate_size=s["shared"], linear_num_key_heads=s["dheads"], linear_num_value_heads=s["dheads"], linear_key_head_dim=128,
                linear_value_head_dim=128, linear_conv_kernel_dim=4, full_attention_interval=3, attn_output_gate=True, partial_rotary_factor=0.25)


def nalasun_kernels(s: dict, iters: int) -> list[dict]:
    """Each kernel of the design beside the like kernel of the closest models. Bytes and FLOPs are the algorithm's: every input read and every output
    written once, and for attention the score, mix and value products over the visible pairs."""
    from types import SimpleNamespace
    from onecat_vllm.ops import cuda as K
    from onecat_vllm.ops import ref
    from onecat_vllm.ops.microbench import _peaks, timeit
    pk, rows = _peaks(), []
    W, H, G, D, E, top = s["width"], s["heads"], s["kv"], s["dim"], s["experts"], s["top"]
    b = lambda *sh: torch.randn(*sh, device="cuda").bfloat16()
    f32 = lambda *sh: torch.randn(*sh, device="cuda")

    def row(kernel, case, who, fn, flops=0.0, nbytes=0.0, n=iters):
        ms = timeit(fn, n)
        t = max(flops / pk["bf16_tflops"] / 1e9, nbytes / pk["hbm_gbs"] / 1e6)
        rows.append(dict(kernel=kernel, case=case, model=who, us=ms * 1e3, roofline_us=t * 1e3, frac_of_roofline=t / ms))

    wide = K.talk_row(H, G, D)
    for case, n, q, S in (("prefill", 1, PREFILL, PREFILL), ("decode", DECODE_REQS, 1, DECODE_CTX)):
        T = n * q
        md, nblk = _meta(n, q, S)
        md.is_uniform_decode = case == "decode"
        pairs = n * sum(range(S - q + 1, S + 1))
        cache, fac, qq, bias, mix = b(nblk, 1, G, 16, wide) * 0.5, torch.ones(nblk, 16, device="cuda"), b(T, H, wide) * 0.1, torch.rand(2, H, device="cuda"), b(H, H) * 0.2
        cost = lambda mixed, tensors: (2.0 * H * pairs * (2 * D + (H if mixed else 0)), 2.0 * (n * S * G * D * tensors + 2 * T * H * D))
        row("attention", case, "nalasun, shared keys, mixed heads", lambda: K.talk_attention(qq, cache, fac, md, bias, mix, D), *cost(True, 1))
        x, out, table = b(T, H, D), torch.empty(T, H, D, dtype=torch.bfloat16, device="cuda"), f32(H, BIAS_MAX + 1)
        row("attention", case, "gabisun, shared keys, distance bias", lambda: K.paged_attention(x, cache, md, D ** -0.5, out=out, bias_table=table), *cost(False, 1))
        del cache
        md.attn_plan = None
        kv = b(nblk, 2, G, 16, D) * 0.5
        row("attention", case, "qwen3-next, plain", lambda: K.paged_attention(x, kv, md, D ** -0.5, out=out), *cost(False, 2))
        del kv
    for case, n, q in (("prefill", 1, PREFILL), ("decode", DECODE_REQS, 1)):
        T = n * q
        md, _ = _meta(n, q, q)
        md.state_slots = torch.arange(n, device="cuda", dtype=torch.int32)
        md.has_initial_state = torch.ones(n, device="cuda", dtype=torch.int32)
        md.is_uniform_decode = case == "decode"
        cx, cw, cs = b(T, W), b(W, 4), b(n, 3, W)
        row("input convolution", case, "nalasun", lambda: K.causal_conv(cx, cw, None, cs, md, False, True), nbytes=4.0 * T * W + 12.0 * n * W)
        # matrix states: the products of the chunked form with 64 tokens (two with the state, one inside the chunk), or the state's traffic
        cost = lambda h, d, v, extra: (4.0 * T * h * (d * v + 32 * (d + v)), 2.0 * T * h * (2 * d + 3 * v) + extra + 8.0 * n * h * d * v)
        h, d = s["dheads"], s["ddim"]
        x, a, st, wt, gate, nw, conv = b(T, 3 * h * d + h), f32(T, h * d), f32(n, h, d, d), b(3 * h * d, 4), b(T, h * d), b(d), b(n, 3, 3 * h * d)
        al, dtb = f32(h), f32(h * d)

        def delta():
            y = K.causal_conv(x[:, : 3 * h * d], wt, None, conv, md, True, False)
            return K.gated_norm(K.channel_delta(y, a, x[:, 3 * h * d:], al, dtb, st, md, h, h, d, d), gate, nw, 1e-5, h, False)
        row("recurrence", case, f"nalasun channel delta {d}x{d} with convolution, head norm and gate", delta, *cost(h, d, d, 4.0 * T * h * d))
        y = K.causal_conv(x[:, : 3 * h * d], wt, None, conv, md, True, False)
        row("recurrence", case, f"nalasun channel delta {d}x{d} alone", lambda: K.channel_delta(y, a, x[:, 3 * h * d:], al, dtb, st, md, h, h, d, d), *cost(h, d, d, 4.0 * T * h * d))
        gc_, gs, gx, ga, gw, gz, gn = b(n, 3 * h * 128, 3), f32(n, h, 128, 128), b(T, 3 * h * 128), b(T, h), b(3 * h * 128, 4), b(T, h * 128), b(128)
        row("recurrence", case, "qwen3-next Gated-DeltaNet 128x128 with convolution, head norm and gate", lambda: K.rms_norm_gated(
            K.gdn_forward(gx, ga, ga, gw, al, al, gc_, gs, md, h, h, 128, 128).reshape(T, h * 128), gz, gn, 1e-5, h), *cost(h, 128, 128, 0.0))
        mh, mv, N, mg = s["mheads"], s["mdim"], s["state"], s["groups"]
        inner, ch = mh * mv, mh * mv + 2 * mg * N
        mx, mw, mb, mc, ms, mn = b(T, inner + ch + mh), b(ch, 4), b(ch), b(n, 3, ch), f32(n, mh, N, mv), b(inner)
        mal, mdt, msk = f32(mh), f32(mh), f32(mh)
        mcost = (4.0 * T * mh * (N * mv + 32 * mv) + 4.0 * T * mg * 32 * N, 2.0 * T * (3 * inner + 2 * mg * N) + 8.0 * n * mh * N * mv)

        def ssm():
            y = K.causal_conv(mx[:, inner: inner + ch], mw, mb, mc, md, True, False)
            return K.gated_norm(K.mamba2(y, mx[:, inner + ch:], mal, mdt, msk, ms, md, mh, mg, N, mv, (0.0, float("inf"))), mx[:, :inner], mn, 1e-5, mg, True)
        row("recurrence", case, f"nalasun Mamba-2 {N}x{mv} x {mh} with convolution, gate and norm", ssm, *mcost)
        my = K.causal_conv(mx[:, inner: inner + ch], mw, mb, mc, md, True, False)
        row("recurrence", case, f"nalasun Mamba-2 {N}x{mv} x {mh} alone", lambda: K.mamba2(my, mx[:, inner + ch:], mal, mdt, msk, ms, md, mh, mg, N, mv, (0.0, float("inf"))), *mcost)
        row("recurrence", case, f"Mamba-2 {N}x{mv} x {mh} alone as PyTorch operations", lambda: ref.mamba2(my, mx[:, inner + ch:], mal, mdt, msk, ms, md, mh, mg, N, mv), *mcost, n=3)
        go = b(T, h * d)
        row("gated norm", case, "nalasun, sigmoid gate", lambda: K.gated_norm(go, gate, nw, 1e-5, h, False), nbytes=6.0 * T * h * d)
        row("gated norm", case, "nalasun, SiLU gate ahead", lambda: K.gated_norm(mx[:, :inner], mx[:, inner: 2 * inner], mn, 1e-5, mg, True), nbytes=6.0 * T * inner)
        row("gated norm", case, "qwen3-next", lambda: K.rms_norm_gated(gz, gx[:, : h * 128], gn, 1e-5, h), nbytes=6.0 * T * h * 128)
    for T in (PREFILL, DECODE_REQS):
        part, x32, w, res = b(T, W), f32(T, W), b(W), b(T, W)
        row("norm", T, "nalasun join", lambda: K.stream_join(part, x32, None, None, (1, w, None, 1e-5, False), torch.bfloat16), nbytes=12.0 * T * W)
        row("norm", T, "add + rms norm", lambda: K.rms_norm(part, w, 1e-5, res, False), nbytes=8.0 * T * W)
        slot = torch.arange(T, device="cuda", dtype=torch.int32)
        ids, emb, pos = torch.randint(0, VOCAB, (T,), device="cuda", dtype=torch.int32), b(VOCAB, W), b(2 * PREFILL, W)
        row("embedding", T, "nalasun, token and position rows", lambda: K.embed_stream(ids, emb, 1.0, None, None, (0, 0), torch.bfloat16, rows=pos, positions=slot), nbytes=8.0 * T * W)
        row("embedding", T, "qwen3-next (PyTorch)", lambda: torch.nn.functional.embedding(ids, emb), nbytes=4.0 * T * W)
        qk, gain, cache, fac = b(T, (H + G) * D), f32(H * D), b(T // 16 + 1, 1, G, 16, wide), f32(T // 16 + 1, 16)
        row("norms + insert", T, "nalasun", lambda: K.talk_prepare(qk, gain, 1e-5, (0.1, 4096), slot, cache, fac, slot, H, G, D), nbytes=4.0 * T * (H + G) * D)
        k2, c2, cs2, nw2 = b(T, (H + 2 * G) * D), b(T // 16 + 1, 2, G, 16, D), torch.ones(T, D, device="cuda"), b(D)
        row("norms + insert", T, "qwen3", lambda: K.rope_and_cache(k2[:, : H * D].view(T, H, D), k2[:, H * D: (H + G) * D].view(T, G, D), k2[:, (H + G) * D:].view(T, G, D),
                                                                 slot, cs2, c2, slot, D, nw2, nw2, 1e-5, False), nbytes=4.0 * T * (H + 2 * G) * D)
        rc = SimpleNamespace(num_experts_per_tok=top, n_group=1, topk_group=1, scoring_func="sigmoid", norm_topk_prob=False, routed_scaling_factor=2.0)
        z, zero = f32(T, E), torch.zeros(E, device="cuda")
        row("router", T, "nalasun (sigmoid, fp32 logits)", lambda: K.route(z, rc, zero), nbytes=T * (4.0 * E + 8.0 * top))
        rq, zb = SimpleNamespace(num_experts_per_tok=top, n_group=1, topk_group=1, scoring_func="softmax", norm_topk_prob=True, routed_scaling_factor=1.0), z.bfloat16()
        row("router", T, "qwen3-next (softmax, bf16 logits)", lambda: K.route(zb, rq, None), nbytes=T * (2.0 * E + 8.0 * top))

        def gemm(name, who, N, Kd, **kw):
            wt, xx = (torch.randn(N, Kd, device="cuda") * 0.02).bfloat16(), b(T, Kd)
            out = torch.empty(T, -(-N // 8) * 8, dtype=kw.get("out_dtype", torch.bfloat16), device="cuda")[:, :N]
            row(f"gemm {name}", T, who, lambda: K._gemm(xx, wt, None, None, out, None, N, N, N, 0, K.EPI_STORE, 1), flops=2.0 * T * N * Kd,
                nbytes=2.0 * (N * Kd + T * Kd) + out.element_size() * T * N)
        h, d = s["dheads"], s["ddim"]
        gemm("mixer input", "nalasun q|k", (H + G) * D, W)
        gemm("mixer input", "nalasun delta q|k|v|a|g|b", 3 * h * d + 2 * d + h, W)
        gemm("mixer input", "nalasun Mamba-2", 2 * s["mheads"] * s["mdim"] + 2 * s["groups"] * s["state"] + s["mheads"], W)
        gemm("mixer input", "qwen3-next q|k|v|z", 4 * h * 128, W)
        gemm("low rank", "nalasun decays, fp32 output", h * d, d, out_dtype=torch.float32)
        gemm("low rank", "nalasun gate", h * d, d)
        gemm("router logits", "nalasun, fp32 output", E, W, out_dtype=torch.float32)
        gemm("router logits", "qwen3-next", E, W)
    return rows


def run_nalasun(steps: int, warmup: int, sizes=None, kernels: bool = True, clock_sampler=None) -> None:
    for name, s in NALASUN_SIZES.items():
        if sizes and name not in sizes:
            continue
        clocks = clock_sampler() if clock_sampler else None
        models = {"Nalasun": nalasun_config(s), "Qwen3-Next": nalasun_like(s, "Qwen3NextForCausalLM"), "Granite 4 hybrid": nalasun_like(s, "GraniteMoeHybridForCausalLM")}
        res = {"design": "nalasun", "size": name, "dims": s, "dtype": "bf16", "data": "synthetic: random token ids and weights",
               "workload": f"prefill: one {PREFILL}-token prompt a step; decode: {DECODE_REQS} requests at a context of about {DECODE_CTX}",
               "l2": "model steps stream weights and caches larger than L2; kernels: L2 flushed before every launch",
               "models": {k: model_throughput(m, steps, warmup) for k, m in models.items()}}
        if kernels:
            res["kernels"] = nalasun_kernels(s, max(5, steps // 6))
        if clocks is not None:
            res["clocks"] = clocks.stop()
        print(json.dumps(res), flush=True)


def run_lodevik(steps: int, warmup: int, sizes=None, kernels: bool = True, clock_sampler=None) -> None:
    for name, s in LODEVIK_SIZES.items():
        if sizes and name not in sizes:
            continue
        clocks = clock_sampler() if clock_sampler else None
        models = {"Lodevik": lodevik_config(s), "Gemma-2": lodevik_like(s, "Gemma2ForCausalLM"), "DeepSeek-V2 (dense)": lodevik_like(s, "DeepseekV2ForCausalLM")}
        res = {"design": "lodevik", "size": name, "dims": s, "dtype": "bf16", "data": "synthetic: random token ids and weights",
               "workload": f"prefill: one {PREFILL}-token prompt a step; decode: {DECODE_REQS} requests at a context of about {DECODE_CTX}",
               "l2": "model steps stream weights and caches larger than L2; kernels: L2 flushed before every launch",
               "models": {k: model_throughput(m, steps, warmup) for k, m in models.items()}}
        if kernels:
            res["kernels"] = lodevik_kernels(s, max(5, steps // 6))
        if clocks is not None:
            res["clocks"] = clocks.stop()
        print(json.dumps(res), flush=True)


def run_sepirax(steps: int, warmup: int, sizes=None, kernels: bool = True, clock_sampler=None) -> None:
    for name, s in SEPIRAX_SIZES.items():
        if sizes and name not in sizes:
            continue
        clocks = clock_sampler() if clock_sampler else None
        models = {"Sepirax": sepirax_config(s), "DeepSeek-V2": sepirax_like(s, "DeepseekV2ForCausalLM"), "Qwen3-Next": sepirax_like(s, "Qwen3NextForCausalLM")}
        res = {"design": "sepirax", "size": name, "dims": s, "dtype": "bf16", "data": "synthetic: random token ids and weights",
               "workload": f"prefill: one {PREFILL}-token prompt a step; decode: {DECODE_REQS} requests at a context of about {DECODE_CTX}",
               "l2": "model steps stream weights and caches larger than L2; kernels: L2 flushed before every launch",
               "models": {k: model_throughput(c, steps, warmup) for k, c in models.items()}}
        if kernels:
            res["kernels"] = sepirax_kernels(s, max(5, steps // 6))
        if clocks is not None:
            res["clocks"] = clocks.stop()
        print(json.dumps(res), flush=True)


def run(steps: int, warmup: int, sizes=None, kernels: bool = True, clock_sampler=None) -> None:
    for name, s in SIZES.items():
        if sizes and name not in sizes:
            continue
        clocks = clock_sampler() if clock_sampler else None
        models = {"Gabisun": gabisun_config(s), "Starcoder2": like_config(s, "Starcoder2ForCausalLM"), "Mistral": like_config(s, "MistralForCausalLM")}
        res = {"design": "gabisun", "size": name, "dims": s, "dtype": "bf16", "data": "synthetic: random token ids and weights",
               "workload": f"prefill: one {PREFILL}-token prompt a step; decode: {DECODE_REQS} requests at a context of about {DECODE_CTX}",
               "l2": "model steps stream weights and KV larger than L2; kernels: L2 flushed before every launch",
               "models": {k: model_throughput(c, steps, warmup) for k, c in models.items()}}
        if kernels:
            res["kernels"] = kernel_rows(s, max(5, steps // 6))
        if clocks is not None:
            res["clocks"] = clocks.stop()
        print(json.dumps(res), flush=True)

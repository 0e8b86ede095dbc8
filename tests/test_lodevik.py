"""Lodevik on the CPU path (fp32) against the plain float64 restatement in lodevik_oracle.py: each mechanism alone, whole prompts, decoding
through the paged cache, portions, mixed batches, reuse of pages, greedy generation through the scheduler."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import lodevik_models as M
import lodevik_oracle as O
from gabisun_models import error, replay, tokens
from onecat_vllm import LLM, SamplingParams, ops
from onecat_vllm.config import ModelConfig
from onecat_vllm.engine.replay import TraceReplay
from onecat_vllm.layers.common import RMSNorm, get_rope
from onecat_vllm.loader.weights import lodevik_name
from onecat_vllm.ops import ref

TOL = 2e-5
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
GREEDY = dict(temperature=0.0, ignore_eos=True, detokenize=False)


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)   # tiny matrices
    yield
    torch.set_num_threads(n)


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in M.CONFIGS.items():
        w = M.make_weights(cfg, seed=len(name), sharp=1.3)
        out[name] = (cfg, w, M.save(cfg, w, tmp_path_factory.mktemp(name)))
    return out


def engine(path, max_tokens, **kw):
    return TraceReplay(path, "float32", max_tokens, device="cpu", **kw)


class Meta:
    def __init__(self, bt, qsl, seq):
        t = lambda v: torch.tensor(v, dtype=torch.int32)
        self.block_table, self.query_start_loc, self.seq_lens = bt, t(qsl), t(seq)


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("buckets,muls", [(97, (31, 7)), (2, (1, 1)), (5003, (70001, 90001)), (1, (5, 9))])
def test_embeddings(buckets, muls):
    """Scaled token rows plus bigram rows; the multipliers times token ids do not fit 32 bits."""
    g = torch.Generator().manual_seed(buckets)
    V, W = 70000, 12
    emb = dict(scale=2.5, bigram=dict(buckets=buckets, mul_prev=muls[0], mul_cur=muls[1]))
    w = {"embed": torch.randn(V, W, generator=g), "bigram": torch.randn(buckets + 1, W, generator=g)}
    toks = [69999, 69999, 0, 5, 5, 69998, 3, 0, 0]
    want = O.embed(toks, {k: v.double() for k, v in w.items()}, emb)
    ids, prev = torch.tensor(toks, dtype=torch.int32), torch.tensor([-1] + toks[:-1], dtype=torch.int32)
    x, y = ops.embed_stream(ids, w["embed"], 2.5, prev, w["bigram"], muls)
    assert torch.allclose(x.double(), want, atol=1e-5) and torch.equal(x, y)
    z, _ = ops.embed_stream(ids, w["embed"][ids.long()], 2.5, prev, w["bigram"], muls, gathered=True)
    assert torch.equal(x, z)
    x, y = ops.embed_stream(ids, w["embed"].bfloat16(), 3.0)
    assert torch.equal(x, w["embed"].bfloat16()[ids.long()].float() * 3) and torch.equal(y, x.bfloat16())


def test_join_with_an_output_norm_only():
    g = torch.Generator().manual_seed(0)
    part, x, scale = (torch.randn(5, 24, generator=g), torch.randn(5, 24, generator=g), torch.randn(24, generator=g))
    n = RMSNorm(24, 1e-3)
    n.weight.data.normal_(generator=g)
    y = torch.empty(5, 24, dtype=torch.bfloat16)
    want = x.double() + O.rms(part.double(), 1e-3) * n.weight.double() * scale.double()
    none, x1 = ops.stream_join(part, x.clone(), n, scale, None, copy_out=y)
    assert none is None and torch.allclose(x1.double(), want, atol=1e-5) and torch.equal(y, x1.bfloat16())


def test_gated_gelu():
    from onecat_vllm.layers.mlp import MLP
    g = torch.Generator().manual_seed(1)
    m = MLP(20, 28, None, "m", torch.float32, act="gelu_tanh")
    w = {n: torch.randn(*s, generator=g) for n, s in (("gate", (28, 20)), ("up", (28, 20)), ("down", (20, 28)))}
    m.gate_up_proj.load_weight("weight", w["gate"], 0), m.gate_up_proj.load_weight("weight", w["up"], 1), m.down_proj.load_weight("weight", w["down"])
    x = torch.randn(9, 20, generator=g)
    want = O.feed_forward(x.double(), {k: v.double() for k, v in w.items()}, "")
    assert torch.allclose(m(x).double(), want, atol=1e-3, rtol=1e-5)


@pytest.mark.parametrize("H,G,D,U,rot,width", [(6, 3, 16, 24, 4, 32), (2, 1, 6, 14, 6, 14), (3, 3, 9, 5, 0, 18), (4, 1, 8, 8, 2, 40)])
def test_maps_are_normalised_rotated_and_inserted(H, G, D, U, rot, width):
    """Norm and rotation per map, keys' maps side by side in the cached row, zeros in the padding; a token without a slot goes nowhere else."""
    g = torch.Generator().manual_seed(width)
    T, bs, eps = 9, 4, 1e-3
    x = torch.randn(T, 2 * (H + G) * D + G * U, generator=g)
    qw, kw = torch.randn(D, generator=g), torch.randn(D, generator=g)
    table = get_rope(rot, 64, 100.0, "cpu").cos_sin
    slots = torch.tensor([5, 23, 4, 22, 13, 7, -1, 8, 31])
    pos = torch.tensor([3, 0, 40, 41, 7, 7, 9, 63, 1])
    cache = torch.full((8, 2, G, bs, width), 9.0)
    q = ops.diff_prepare(x, qw, kw, eps, pos, table, cache, slots, H, G, D, U)
    spec = dict(dims=rot, base=100.0)
    xq, xk, xv = x.double().split([2 * H * D, 2 * G * D, G * U], 1)
    finish = lambda v, n, w: O.rotate((O.rms(v.view(T, 2 * n, D), eps) * w.double()).transpose(0, 1), pos, spec).transpose(0, 1)
    assert torch.allclose(q[..., :D].double(), finish(xq, H, qw), atol=1e-5) and not q[..., D:].any()
    wk = finish(xk, G, kw)
    for t in range(T):
        if slots[t] >= 0:
            row = cache[slots[t] // bs, :, :, slots[t] % bs].double()
            for h in range(G):
                for m in range(2):
                    half = row[0, h, m * width // 2: (m + 1) * width // 2]
                    assert torch.allclose(half[:D], wk[t, 2 * h + m], atol=1e-5) and not half[D:].any()
                assert torch.allclose(row[1, h, :U], xv[t, h * U:(h + 1) * U]) and not row[1, h, U:].any()
    used = set(slots.tolist()) | {0}
    rows = cache.permute(0, 3, 1, 2, 4).reshape(32, -1)
    assert (rows[[i for i in range(32) if i not in used]] == 9.0).all()


def paged(k, v, width, bs=16, seed=0):
    """k [S, G, 2, D], v [S, G, U] -> cache [pages, 2, G, bs, width] in shuffled pages and the block table."""
    S, G, _, D = k.shape
    nb = -(-S // bs)
    perm = torch.randperm(nb + 2, generator=torch.Generator().manual_seed(seed))[:nb]
    cache = torch.full((nb + 2, 2, G, bs, width), 5.0, dtype=k.dtype)
    for s in range(S):
        row = torch.zeros(2, G, width, dtype=k.dtype)
        row[0, :, :D], row[0, :, width // 2: width // 2 + D], row[1, :, : v.shape[2]] = k[s, :, 0], k[s, :, 1], v[s]
        cache[perm[s // bs], :, :, s % bs] = row
    return cache, perm.view(1, -1).to(torch.int32)


@pytest.mark.parametrize("H,G,D,U,width", [(6, 3, 16, 24, 32), (2, 1, 6, 14, 14), (3, 3, 9, 5, 24)])
@pytest.mark.parametrize("cap,chunk", [(4.0, 30), (0.0, 0), (9.0, 1), (2.0, 64), (3.0, 1000)])
def test_difference_of_two_maps(H, G, D, U, width, cap, chunk):
    g = torch.Generator().manual_seed(H + U)
    S = 97
    q, k, v = torch.randn(S, H, 2, D, generator=g) * 2, torch.randn(S, G, 2, D, generator=g), torch.randn(S, G, U, generator=g)
    lam, mx = torch.tensor([0.7]), dict(scale=0.4, softcap=cap, mask=dict(size=chunk) if chunk else None, diff=0.3)
    want = O.differential(q.double().permute(1, 2, 0, 3), k.double().permute(1, 2, 0, 3), v.double().permute(1, 0, 2), mx, 0.7, 1e-5).permute(1, 0, 2)
    cache, bt = paged(k, v, width)
    qp = torch.nn.functional.pad(q, (0, width // 2 - D)).reshape(S, 2 * H, width // 2)
    for n in (97, 1, 2, 40, 68):
        got = ops.diff_attention(qp[S - n:], cache, Meta(bt, [0, n], [S]), 0.4, lam, 0.7, 1e-5, U, cap, chunk)
        # a difference that nearly vanishes is normalised noise: compare what is well above rounding
        assert (got.double() - want[S - n:]).abs().max() < 2e-3 and (got.double() - want[S - n:]).abs().mean() < 2e-6


@pytest.mark.parametrize("m", [0, 1])
def test_one_key_stands_out_at_page_and_chunk_edges(m):
    """A query of one map that matches exactly one cached key of that map finds it inside its chunk, wherever it lies, and nowhere else."""
    D, U, bs, S, chunk = 8, 16, 16, 420, 50
    g = torch.Generator().manual_seed(3)
    for i in (0, 15, 16, 49, 50, 51, 99, 100, 149, 399, 400, 419):
        lo = i - i % chunk
        for j in sorted({0, 1, lo - 1, lo, lo + 1, i - 49, i - 16, i - 1, i, i + 1, i - chunk} & set(range(min(i + 2, S)))):
            k, v = torch.randn(S, 1, 2, D, generator=g) * 0.1, torch.randn(S, 1, U, generator=g)
            k[j, 0, m] = torch.randn(D, generator=g) * 3
            cache, bt = paged(k, v, U, bs, seed=j)
            q = torch.zeros(1, 2, D)
            q[0, m] = k[j, 0, m] * 4
            # the other map sees its chunk evenly; without it (lambda 0) or against it the key's value remains
            o = ops.diff_attention(q, cache, Meta(bt, [0, 1], [i + 1]), 1.0, torch.tensor([0.0 if m == 0 else 50.0]), 1.0, 1e-6, U, 0.0, chunk)[0, 0]
            sign = 1 if m == 0 else -1
            assert bool(torch.cosine_similarity(sign * o, v[j, 0], dim=0) > 0.98) == (lo <= j <= i) or i == lo and j == i, (i, j)


def test_latent_sink_and_head_gate():
    """The sink takes weight and gives nothing; the gate is one factor per head; the scores' scale does not touch the sink."""
    g = torch.Generator().manual_seed(5)
    S, H, L, R, bs = 70, 3, 12, 4, 16
    lat = torch.randn(S, L + R, generator=g)
    cache = torch.cat([lat, torch.full((10, L + R), 7.0)]).view(5, bs, L + R)
    q, sink, gate = torch.randn(S, H, L + R, generator=g), torch.tensor([-2.0, 1.0, 6.0]), torch.randn(S, H, generator=g)
    got = ref.mla_decode(q[..., :L], q[..., L:], cache, torch.arange(5, dtype=torch.int32).view(1, -1), torch.tensor([0, S]), torch.tensor([S]), 0.5, L, sink, gate)
    s = torch.einsum("qhd,kd->hqk", q.double(), lat.double()) * 0.5
    want = O.weights(s, O.sees(S), sink.double()) @ lat[:, :L].double() * torch.sigmoid(gate.double()).T.unsqueeze(-1)
    assert torch.allclose(got.double(), want.permute(1, 0, 2), atol=1e-5)


def test_chunked_plain_attention():
    """The chunk mask is an option of ordinary attention as well."""
    g = torch.Generator().manual_seed(6)
    S, Hq, Hkv, D = 90, 4, 2, 16
    q, k, v = (torch.randn(S, h, D, generator=g) for h in (Hq, Hkv, Hkv))
    cache = torch.zeros(6, 2, Hkv, 16, D)
    for s in range(S):
        cache[s // 16, 0, :, s % 16], cache[s // 16, 1, :, s % 16] = k[s], v[s]
    got = ops.paged_attention(q, cache, Meta(torch.arange(6, dtype=torch.int32).view(1, -1), [0, S], [S]), 0.3, chunk=25)
    for h in range(Hq):
        s = (q[:, h].double() @ k[:, h // 2].double().T) * 0.3
        want = O.weights(s.unsqueeze(0), O.sees(S, 25))[0] @ v[:, h // 2].double()
        assert torch.allclose(got[:, h].double(), want, atol=1e-5)


# ------------------------------------------------------------------------------------------------ configuration and loading
def test_config_and_names():
    cfg = M.CONFIGS["mixed"]
    mc = ModelConfig.from_hf_dict(cfg)
    a, b, c, d = (mc.for_layer(i) for i in range(4))
    assert (a.num_attention_heads, a.num_key_value_heads, a.head_dim, a.v_head_dim, a.rotary_dim, a.attn_chunk, a.attn_softcap, a.attn_diff, a.use_mla,
            a.intermediate_size, a.attn_sinks, a.attn_head_gate) == (6, 3, 16, 24, 4, 37, 6.0, 0.3, False, 160, False, False)
    assert (b.use_mla, b.num_attention_heads, b.kv_lora_rank, b.qk_nope_head_dim, b.qk_rope_head_dim, b.v_head_dim, b.q_lora_rank, b.mixer_only_layers,
            b.attn_sinks, b.attn_head_gate, b.attn_diff) == (True, 4, 40, 24, 8, 16, 0, True, True, True, None)
    assert c.intermediate_size == 72 and not c.mixer_only_layers and d.mixer_only_layers and d.attn_diff == 0.8 and d.rotary_dim == 48
    assert (mc.embed_scale, mc.bigram, mc.logit_scale, mc.rms_norm_eps, mc.tie_word_embeddings) == (2.0, (301, 1009, 613), 0.8, 1e-5, True)
    assert mc.release_window() == (0, 0) and ModelConfig.from_hf_dict(M.CONFIGS["chunks"]).release_window() == (50, 0)
    assert lodevik_name("l12.mix.lq2") == "model.layers.12.self_attn.lq2" and lodevik_name("l0.norm1") == "model.layers.0.post_attention_layernorm.weight"
    assert lodevik_name("bigram") == "model.bigram.weight" and lodevik_name("l3.mix.dkv.norm") == "model.layers.3.self_attn.kv_a_layernorm.weight"
    assert lodevik_name("l1.mlp.gate") == "model.layers.1.mlp.gate_proj.weight" and lodevik_name("l1.mix.new") == "l1.mix.new"
    l0, l1 = cfg["layers"][:2]
    for bad in (dict(l0, type="conv"), dict(l0, mlp=dict(kind="moe", ff=8)), dict(l1, mixer=dict(l1["mixer"], rot_dim=16)),
                dict(l0, mixer=dict(l0["mixer"], rot=dict(base=10.0, dims=5))), dict(l0, mixer=dict(l0["mixer"], rot=dict(base=10.0, dims=18))),
                dict(l0, mixer=dict(l0["mixer"], kv_heads=4))):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(dict(cfg, layers=[bad]))


def test_every_tensor_of_a_checkpoint_is_used(models):
    from onecat_vllm.loader.weights import iter_safetensors, load_weights
    from onecat_vllm.models import build_model
    for name, (cfg, w, path) in models.items():
        mc = ModelConfig.from_pretrained(path, dtype=torch.float32)
        with torch.device("cpu"):
            m = build_model(mc)
        assert len(load_weights(m, iter_safetensors(path))) == len(w), name
        params = sum(p.numel() for p in m.parameters())
        assert params == sum(v.numel() for v in w.values()) + (m.model.embed_tokens.padded - cfg["vocab"]) * cfg["width"], name


def test_lambda_is_one_number_per_layer(models):
    cfg, w, path = models["mixed"]
    run = engine(path, 64)
    layers = run.core.executor.worker.runner.model.model.layers
    for i in (0, 3):
        want = O.difference_factor({k: v.double() for k, v in w.items()}, f"l{i}.mix.", cfg["layers"][i]["mixer"]["diff"])
        assert layers[i].self_attn.lam.item() == pytest.approx(want.item(), abs=1e-6)
    shapes = [tuple(c.shape[1:]) for c in run.core.executor.worker.runner.kv_caches]
    assert shapes == [(2, 3, 16, 32), (16, 48), (16, 80), (2, 1, 16, 96)]
    run.close()


# ------------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_whole_prompt(models, name):
    cfg, w, path = models[name]
    toks = tokens(cfg, 150)
    run = engine(path, 160)
    got = replay(run, {"a": toks}, [[("a", 150)]])["a"]
    assert error(got, O.forward(cfg, w, toks)[0]) < TOL
    run.close()


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_portions_and_decoding(models, name):
    cfg, w, path = models[name]
    toks = tokens(cfg, 110, 1)
    want = O.forward(cfg, w, toks)[0]
    run = engine(path, 112)
    for sizes in ([1] * 110, [2] * 55, [3, 60, 1, 1, 2, 43], [17] * 7, [37, 37, 36], [70] + [1] * 40):
        got = replay(run, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert error(got, want) < TOL, sizes[:4]
    run.close()


@pytest.mark.parametrize("name", ["mixed", "chunks"])
def test_mixed_batches_reuse_pages(models, name):
    """Unequal requests together, each left out of some steps, in a pool for the live ones only: logits equal those alone."""
    cfg, w, path = models[name]
    seqs = {f"r{i}": tokens(cfg, n, 10 + i) for i, n in enumerate((90, 1, 47, 64, 16, 70, 33, 80))}
    run = engine(path, 256)
    steps = [[("r0", 40), ("r1", 1), ("r2", 2)], [("r2", 1), ("r3", 63)], [("r0", 1), ("r3", 1), ("r2", 44), ("r4", 3)], [("r4", 1), ("r0", 17)],
             [("r5", 50), ("r4", 12), ("r0", 1)]] + [[("r0", 2), ("r5", 1)]] * 15 + [[("r0", 99), ("r5", 99), ("r6", 5)], [("r6", 28), ("r7", 2)]] + \
            [[("r7", 1)]] * 30 + [[("r7", 68)]]
    got = replay(run, seqs, steps)
    for k, t in seqs.items():
        assert error(got[k], O.forward(cfg, w, t)[0]) < TOL, k
    assert run.core.scheduler.kv_cache_manager.block_pool.get_num_free_blocks() == 256 // 16
    again = replay(run, {"r0": seqs["r5"]}, [[("r0", 30)], [("r0", 40)]])["r0"]   # the same ids may come back as new requests
    assert error(again, got["r5"]) < TOL
    run.close()


def test_pages_outside_every_chunk_are_given_back(models):
    cfg, w, path = models["chunks"]
    toks = tokens(cfg, 400, 4)
    run = engine(path, 400)
    got = replay(run, {"a": toks}, [[("a", 200)]] + [[("a", 20)]] * 10, end=False)["a"]
    assert error(got, O.forward(cfg, w, toks)[0]) < TOL
    kept = sum(not b.is_null for b in run.core.scheduler.kv_cache_manager.req_to_blocks["a"])
    assert kept <= (50 + 128 + 20) // 16 + 3
    run.close()


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_greedy_generation_through_the_scheduler(models, name):
    cfg, w, path = models[name]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=128, max_num_batched_tokens=32, max_num_seqs=3)
    prompts = [tokens(cfg, n, 30 + n) for n in (50, 3, 1, 41)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(max_tokens=16, **GREEDY))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 16)


def test_the_token_ahead_is_known_behind_a_cached_prefix(models):
    """Requests that share whole pages of their prompts compute only what follows: the bigram there reaches back into the shared part."""
    cfg, w, path = models["wide"]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=128, enable_prefix_caching=True)
    base, hits = tokens(cfg, 48, 3), []
    for tail in ([5], [9, 9], tokens(cfg, 20, 4)):
        o = llm.generate([{"prompt_token_ids": base + tail}], SamplingParams(max_tokens=8, **GREEDY))[0]
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, base + tail, 8)
        hits.append(o.num_cached_tokens)
    assert hits == [0, 48, 48]


@pytest.mark.parametrize("overlap", [True, False])
def test_preemption_and_overlapped_steps(models, overlap):
    """Few pages: requests are thrown out and recomputed. With overlapped steps a decoded token is on the device only when the next step's
    inputs are staged; the one ahead of it is known."""
    cfg, w, path = models["mixed"]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=96, max_num_seqs=4, num_gpu_blocks_override=11, async_scheduling=overlap)
    prompts = [tokens(cfg, 20, 60 + i) for i in range(4)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(max_tokens=40, **GREEDY))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 40)


def test_ngram_drafts_are_verified_like_decoded_tokens(models):
    cfg, w, path = models["mixed"]
    p = tokens(cfg, 12, 5) * 3
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=128,
              speculative_config=dict(method="ngram", num_speculative_tokens=3, prompt_lookup_max=3, prompt_lookup_min=1))
    o = llm.generate([{"prompt_token_ids": p}], SamplingParams(max_tokens=30, **GREEDY))[0]
    assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 30)


def test_trace_runner_program(models, tmp_path):
    cfg, w, path = models["odd"]
    toks = tokens(cfg, 30, 3)
    lines = [dict(step=0, entries=[dict(id="a", tokens=toks[:20], want=[3, 19]), dict(id="b", tokens=toks[:5], want=[])], end=["b"]),
             dict(step=1, entries=[dict(id="a", tokens=toks[20:29], want=[])], end=[]),
             dict(step=2, entries=[dict(id="b", tokens=toks[:1], want=[0]), dict(id="a", tokens=toks[29:], want=[0])], end=["a", "b"])]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens",
                        "128", "--device", "cpu"], input="".join(json.dumps(l) + "\n" for l in lines), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    want = O.forward(cfg, w, toks)[0]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / n).read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
    assert error(read("0.f32"), want[[3, 19]]) < TOL
    assert error(read("2.f32"), torch.stack([want[0], want[29]])) < TOL


def test_random_weights_without_a_checkpoint():
    llm = LLM(hf_config=M.CONFIGS["mixed"], dtype="float32", device="cpu", max_model_len=64)
    o = llm.generate([{"prompt_token_ids": [1, 2, 3]}], SamplingParams(max_tokens=4, **GREEDY))
    assert len(o[0].outputs[0].token_ids) == 4


def test_prompt_given_as_vectors(models):
    """Vectors take the place of the stream's start; the first token behind them has no previous token, the next ones have."""
    from onecat_vllm.inputs import EmbedsPrompt
    cfg, w, path = models["latents"]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=64)
    w64 = {k: v.double() for k, v in w.items()}
    p, out = tokens(cfg, 9, 2), []
    start = O.embed(p, w64, cfg["embedding"])
    for _ in range(6):
        x = torch.cat([start, O.embed(out, w64, cfg["embedding"])]) if out else start
        for i, lc in enumerate(cfg["layers"]):
            x = O.layer(x, w64, i, lc, cfg["norm"]["eps"])
        out.append(int(((O.rms(x[-1], cfg["norm"]["eps"]) * w64["final.norm"]) @ w64["embed"].T).argmax()))
    got = llm.generate([EmbedsPrompt(prompt_embeds=start.float())], SamplingParams(max_tokens=6, **GREEDY))[0].outputs[0].token_ids
    assert list(got) == out


# ------------------------------------------------------------------------------------------------ what the comparisons would catch
def _mutate(cfg, w, what):
    cfg, w = copy.deepcopy(cfg), {k: v.clone() for k, v in w.items()}
    emb = cfg["embedding"]
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}.mix."
        if what == "scale":
            m["scale"] *= 1.02
        if what == "base":
            m["rot"]["base"] *= 1.1
        if what == "layer scale":
            w[f"l{i}.ls1"] *= 1.05
        if l["type"] == "latent_attention":
            if what == "sink":
                w[p + "sink"] -= 30
            if what == "head gate":
                w[p + "g"] *= 1.1
            if what == "shared key":
                w[p + "dkv"][m["kv_rank"]:] *= 1.05
        else:
            if what in ("softcap", "diff"):
                m[what] *= 1.1
            if what == "lambda":
                w[p + "lq2"] *= 1.1
            if what == "chunk longer":
                m["mask"]["size"] += 1
            if what == "chunk shorter":
                m["mask"]["size"] -= 1
            if what == "no chunk":
                m["mask"] = None
            if what == "swapped maps":
                D = m["dim"]
                w[p + "k"] = w[p + "k"].view(m["kv_heads"], 2, D, -1).flip(1).reshape(w[p + "k"].shape)
    if what == "embed":
        emb["scale"] *= 1.02
    if what == "previous token":
        emb["bigram"]["mul_prev"] += 1
    if what == "first token":
        w["bigram"][-1] *= 0.5
    if what == "eps":
        cfg["norm"]["eps"] *= 100
    return cfg, w


@pytest.mark.parametrize("what", ["scale", "base", "layer scale", "sink", "head gate", "shared key", "softcap", "diff", "lambda", "chunk longer", "chunk shorter",
                                  "no chunk", "swapped maps", "embed", "previous token", "first token", "eps"])
def test_mistakes_show_in_the_logits(models, what):
    """A mistake planted in the restatement moves the logits by far more than the tolerance, so the comparisons above would find the same
    mistake in the engine."""
    cfg, w, _ = models["mixed"]
    toks = tokens(cfg, 110, 7)
    assert error(O.forward(*_mutate(cfg, w, what), toks)[0], O.forward(cfg, w, toks)[0]) > (2 if what == "eps" else 50) * TOL


@pytest.mark.timeout(300)
def test_two_tensor_parallel_ranks(tmp_path):
    """Heads of both mixers, their sinks and gates, the feed-forward's columns and the vocabulary are split over the ranks; the latents and the
    bigram rows are on both."""
    cfg = M.config(64, 91, [M.attn(4, 2, 8, 12, 4, 20, 48), M.latent(6, 16, 8, 24, 40, 32), M.attn(2, 1, 16, 16, 16, 50, None)])
    w = M.make_weights(cfg, 3, sharp=1.3)
    llm = LLM(model=M.save(cfg, w, tmp_path), dtype="float32", device="cpu", max_model_len=128, tensor_parallel_size=2, distributed_executor_backend="mp")
    prompts = [tokens(cfg, n, n) for n in (5, 60)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(max_tokens=12, **GREEDY))
    llm.shutdown()
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 12)


def test_combinations_that_are_not_served_are_refused(models):
    _, _, path = models["odd"]
    for kw in (dict(pipeline_parallel_size=2), dict(tensor_parallel_size=2), dict(kv_cache_dtype="fp8"),
               dict(speculative_config=dict(method="mtp", num_speculative_tokens=1))):
        with pytest.raises(ValueError):
            LLM(model=path, dtype="float32", device="cpu", max_model_len=64, **kw)

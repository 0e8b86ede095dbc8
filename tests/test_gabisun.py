"""Gabisun on the CPU path (fp32) against the plain float64 restatement in gabisun_oracle.py: each mechanism alone, whole prompts, decoding
through the paged cache, portions, mixed batches, page reuse, greedy generation through the scheduler."""
import json
import subprocess
import sys
import os

import pytest
import torch

import gabisun_models as M
import gabisun_oracle as O
from onecat_vllm import LLM, SamplingParams
from onecat_vllm import ops
from onecat_vllm.config import ModelConfig
from onecat_vllm.core.kv_cache_manager import KVCacheManager
from onecat_vllm.engine.replay import TraceReplay
from onecat_vllm.loader.weights import gabisun_name
from onecat_vllm.ops import ref

TOL = 2e-5
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, cfg in M.CONFIGS.items():
        w = M.make_weights(cfg, seed=len(name), sharp=1.5)
        out[name] = (cfg, w, M.save(cfg, w, tmp_path_factory.mktemp(name)))
    return out


def engine(path, max_tokens, **kw):
    return TraceReplay(path, "float32", max_tokens, device="cpu", **kw)


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("buckets,top", [(8, 40), (32, 128), (16, 128), (16, 64), (6, 5), (2, 7), (12, 1000), (10, 81)])
def test_distance_buckets(buckets, top):
    got = ref.distance_buckets(buckets, top)
    assert got == [O.distance_bucket(n, buckets, top) for n in range(top + 1)]
    assert got[-1] == buckets - 1 and got == sorted(got)
    assert O.distance_bucket(10 * top, buckets, top) == buckets - 1


def test_distance_buckets_at_exact_edges():
    # 16 rows up to 128: half 8, and 128 / 8 = 16, so the steps fall exactly on 8 * 2^(m/2): distances 16, 32 and 64 begin a bucket
    b = ref.distance_buckets(16, 128)
    assert [b[n] - b[n - 1] for n in (16, 32, 64)] == [1, 1, 1] and (b[16], b[32], b[64], b[128]) == (10, 12, 14, 15)
    with pytest.raises(ValueError):
        ref.distance_buckets(16, 8)


class Norm:
    def __init__(self, w, b, eps, kind):
        self.weight, self.bias, self.eps, self.plain, self.gemma = w, b, eps, kind == 2, False


def test_stream_join_matches_separate_steps():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g)
    part, x, w1, b1, w2, b2, ls, add = r(5, 24), r(5, 24), r(24), r(24), r(24), r(24), r(24), r(24)
    x0 = x.clone()
    copy = torch.empty(5, 48)
    y, x1 = ops.stream_join(part, x, Norm(w1, b1, 1e-3, 2), ls, Norm(w2, b2, 1e-3, 2), out_dtype=torch.float32, add=add, copy_out=copy[:, :24])
    want = x0.double() + ls * O.layer_norm(part.double(), w1, b1, 1e-3) + add
    assert x1 is x and torch.allclose(x1.double(), want, atol=1e-5) and torch.equal(copy[:, :24], x1)
    assert torch.allclose(y.double(), O.layer_norm(want, w2, b2, 1e-3), atol=1e-5)
    y, x1 = ops.stream_join(part, None, None, None, Norm(w2, None, 1e-3, 1), out_dtype=torch.float32)
    assert torch.equal(x1, part) and torch.allclose(y, part / torch.sqrt(part.pow(2).mean(-1, keepdim=True) + 1e-3) * w2, atol=1e-5)
    assert ops.stream_join(part, x0, None, None, None)[0] is None


def paged(k, bs=16, spare=3):
    """A sequence's keys ``[S, G, D]`` in a one-tensor paged cache whose pages lie in no particular order."""
    S, G, D = k.shape
    nb = -(-S // bs)
    perm = torch.randperm(nb + spare, generator=torch.Generator().manual_seed(S))[:nb]
    cache = torch.full((nb + spare, 1, G, bs, D), 3.0)
    ops.kv_insert(k, cache, torch.tensor([int(perm[i // bs]) * bs + i % bs for i in range(S)], dtype=torch.int32))
    return cache, perm.to(torch.int32).view(1, -1)


class Meta:
    def __init__(self, bt, nq, S):
        self.block_table, self.query_start_loc, self.seq_lens = bt, torch.tensor([0, nq], dtype=torch.int32), torch.tensor([S], dtype=torch.int32)


@pytest.mark.parametrize("size,keep,S,nq", [(20, 3, 70, 70), (20, 3, 70, 1), (1, 0, 40, 40), (16, 16, 50, 2), (7, 30, 60, 60), (500, 9, 45, 45), (33, 1, 100, 5)])
def test_attention_op_against_oracle(size, keep, S, nq):
    H, G, D, B, top = 6, 2, 8, 8, 40
    g = torch.Generator().manual_seed(size + keep)
    q, k = torch.randn(S, H, D, generator=g), torch.randn(S, G, D, generator=g)
    rel, sink, gate = torch.randn(B, H, generator=g), torch.randn(H, generator=g), torch.randn(S, H, generator=g)
    cache, bt = paged(k)
    table = rel[torch.tensor(ref.distance_buckets(B, top))].t().contiguous()
    got = ops.paged_attention(q[S - nq:], cache, Meta(bt, nq, S), 0.7, window=size, sinks=sink, keep=keep, bias_table=table, gate=gate[S - nq:])
    kk = k.permute(1, 0, 2).repeat_interleave(H // G, 0).double()
    s = q.permute(1, 0, 2).double() @ kk.transpose(1, 2) * 0.7 + O.bias_matrix(S, rel.double(), top)
    s = s.masked_fill(~O.visibility(S, dict(size=size, keep_first=keep)), -torch.inf)
    want = (O.sink_softmax(s, sink.double()) @ kk * torch.sigmoid(gate.double()).T.unsqueeze(-1)).permute(1, 0, 2)[S - nq:]
    assert torch.allclose(got.double(), want, atol=1e-5)


def test_one_key_stands_out_at_every_edge():
    """A query that matches exactly one key: the output is that key when it is visible and unrelated to it when it is one token too far."""
    S, D, size, keep = 80, 16, 24, 5
    g = torch.Generator().manual_seed(3)
    for i in (23, 24, 28, 29, 47, 48, 79):
        for j in sorted({0, 4, 5, 15, 16, i - size, i - size + 1, i - size + 2, i}):
            if not 0 <= j <= i:
                continue
            k = torch.randn(S, 1, D, generator=g) * 0.1
            k[j] = torch.randn(1, D, generator=g) * 3
            q = k[j].view(1, 1, D) * 4
            cache, bt = paged(k[: i + 1])
            o = ops.paged_attention(q, cache, Meta(bt, 1, i + 1), 1.0, window=size, keep=keep)[0, 0]
            seen = torch.cosine_similarity(o, k[j, 0], dim=0) > 0.99
            assert bool(seen) == O.visible(i, j, dict(size=size, keep_first=keep)), (i, j)


def test_sink_takes_mass_once_and_has_no_value():
    q, k = torch.zeros(1, 1, 4), torch.ones(2, 1, 4)
    cache, bt = paged(k)
    o = ops.paged_attention(q, cache, Meta(bt, 1, 2), 1.0, sinks=torch.tensor([1.5]))
    assert torch.allclose(o, torch.full_like(o, 2 / (2 + 2.718281828 ** 1.5)), atol=1e-6)


# ------------------------------------------------------------------------------------------------ configuration and loading
def test_config_and_names():
    cfg = M.CONFIGS["mixed"]
    mc = ModelConfig.from_hf_dict(cfg)
    assert mc.layer_runs() == [(0, -1), (1, 0), (2, 0), (1, 1), (2, 1), (1, 2), (2, 2), (3, -1)]
    assert mc.layer_runs() == [(i, -1 if t is None else t) for i, t in O.layer_runs(cfg)]
    assert [mc.for_layer(i).num_attention_heads for i in range(4)] == [4, 6, 8, 2] and mc.for_layer(2).attn_window_keep == 9
    assert mc.for_layer(1).mixer_only_layers and mc.release_window() == (300, 9)
    assert gabisun_name("l12.norm2b.b") == "model.layers.12.post_feedforward_layernorm.bias"
    assert gabisun_name("l0.mix.rel") == "model.layers.0.self_attn.rel_bias" and gabisun_name("loop.step") == "model.loop_step"
    for bad in (dict(type="conv"), dict(mixer=dict(cfg["layers"][0]["mixer"], vdim=8)), dict(mlp=dict(kind="moe", ff=8))):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(dict(cfg, layers=[dict(cfg["layers"][0], **bad)]))
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(dict(cfg, loop=dict(start=2, stop=9, times=1)))


def test_every_pass_has_its_own_pages_and_values_are_stored_once(models):
    cfg, w, path = models["mixed"]
    run = engine(path, 64)
    r = run.core.executor.worker.runner
    assert [tuple(c.shape[1:3]) + (c.shape[4],) for c in r.kv_caches] == [(1, 2, 32)] + [(1, 3, 16), (1, 1, 64)] * 3 + [(1, 2, 48)]
    assert len({c.data_ptr() for c in r.kv_caches}) == 8
    run.close()


# ------------------------------------------------------------------------------------------------ the model
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_whole_prompt(models, name):
    cfg, w, path = models[name]
    toks = M.tokens(cfg, 150)
    run = engine(path, 160)
    got = M.replay(run, {"a": toks}, [[("a", 150)]])["a"]
    assert M.error(got, O.forward(cfg, w, toks)[0]) < TOL
    run.close()


@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_portions_and_decoding(models, name):
    cfg, w, path = models[name]
    toks = M.tokens(cfg, 140, 1)
    want = O.forward(cfg, w, toks)[0]
    run = engine(path, 144)
    for sizes in ([1] * 140, [2] * 70, [3, 100, 1, 1, 2, 33], [17] * 9, [64, 64, 12], [90] + [1] * 50):
        got = M.replay(run, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert M.error(got, want) < TOL, sizes[:4]
    run.close()


def test_mixed_batches_reuse_pages(models):
    """Unequal requests together, each left out of some steps, in a pool that only holds the live ones: logits equal those alone."""
    cfg, w, path = models["mixed"]
    seqs = {f"r{i}": M.tokens(cfg, n, 10 + i) for i, n in enumerate((130, 1, 47, 64, 16, 99, 33, 130))}
    run = engine(path, 336)
    steps = [[("r0", 40), ("r1", 1), ("r2", 2)], [("r2", 1), ("r3", 63)], [("r0", 1), ("r3", 1), ("r2", 44), ("r4", 3)], [("r4", 1), ("r0", 17)],
             [("r5", 50), ("r4", 12), ("r0", 1)]] + [[("r0", 2), ("r5", 3)]] * 15 + [[("r0", 99), ("r5", 99), ("r6", 5)], [("r6", 28), ("r7", 2)]] + \
            [[("r7", 1)]] * 60 + [[("r7", 68)]]
    got = M.replay(run, seqs, steps)
    for k, t in seqs.items():
        assert M.error(got[k], O.forward(cfg, w, t)[0]) < TOL, k
    pool = run.core.scheduler.kv_cache_manager.block_pool
    assert pool.get_num_free_blocks() == 336 // 16
    # the same ids may come back as new requests
    again = M.replay(run, {"r0": seqs["r5"]}, [[("r0", 30)], [("r0", 69)]])["r0"]
    assert M.error(again, got["r5"]) < TOL
    run.close()


def test_pages_outside_the_window_are_given_back(models):
    """Long decoding in a pool smaller than the sequence: only the window and the kept first tokens stay."""
    cfg = M.config(64, 50, [M.layer(2, 1, 16, 40, 5, 32), M.layer(2, 2, 16, 70, 3, 32)], loop=(0, 2, 2))
    w = M.make_weights(cfg, 5, sharp=1.5)
    import tempfile
    with tempfile.TemporaryDirectory() as d:
        path = M.save(cfg, w, d)
        run = engine(path, 640)
        m = run.core.scheduler.kv_cache_manager
        assert (m.sliding_window, m.window_keep_blocks) == (70, 4)
        toks = M.tokens(cfg, 600)
        want = O.forward(cfg, w, toks)[0]
        got = M.replay(run, {"a": toks}, [[("a", 300)]] + [[("a", 1)]] * 300, end=False)["a"]
        assert M.error(got, want) < TOL
        live = [i for i, b in enumerate(m.req_to_blocks["a"]) if not b.is_null]
        assert live[:4] == [0, 1, 2, 3] and len(live) < 22, live
        run.close()


def test_first_tokens_stay_allocated():
    m = KVCacheManager(64, 16, 2048, enable_caching=False, sliding_window=32, window_keep=65)
    assert m.window_keep_blocks == 8
    blocks = m.block_pool.get_new_blocks(30)
    m._free_out_of_window(blocks, 470)
    assert [b.is_null for b in blocks] == [False] * 8 + [True] * 11 + [False] * 11


@pytest.mark.parametrize("name", ["mixed", "plain", "loop_all"])
def test_greedy_generation_through_the_scheduler(models, name):
    cfg, w, path = models[name]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=256, max_num_batched_tokens=32, max_num_seqs=3)
    prompts = [M.tokens(cfg, n, 30 + n) for n in (50, 3, 1, 41)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True, detokenize=False))
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 24)


def test_prefix_cache_and_preemption_keep_the_tokens(models):
    cfg, w, path = models["mixed"]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=128, max_num_seqs=4, num_gpu_blocks_override=14)
    shared = M.tokens(cfg, 40, 50)
    prompts = [shared + M.tokens(cfg, 5, 60 + i) for i in range(4)]
    sp = SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True, detokenize=False)
    for _ in range(2):
        outs = llm.generate([{"prompt_token_ids": p} for p in prompts], sp)
        for p, o in zip(prompts, outs):
            assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 40)


def test_replay_refuses_bad_steps(models):
    cfg, w, path = models["plain"]
    run = engine(path, 64)
    for bad in ([dict(id="a", tokens=[cfg["vocab"]], want=[])], [dict(id="a", tokens=[1], want=[1])], [dict(id="a", tokens=[1], want=[])] * 2):
        with pytest.raises(ValueError):
            run.step(bad)
        run.core.scheduler.finish_requests("a")
    with pytest.raises((RuntimeError, ValueError)):
        run.step([dict(id="b", tokens=[1] * 80, want=[])])
    run.close()


def test_trace_runner_program(models, tmp_path):
    cfg, w, path = models["plain"]
    toks = M.tokens(cfg, 30, 3)
    lines = [dict(step=0, entries=[dict(id="a", tokens=toks[:20], want=[3, 19]), dict(id="b", tokens=toks[:5], want=[])], end=["b"]),
             dict(step=1, entries=[dict(id="a", tokens=toks[20:29], want=[])], end=[]),
             dict(step=2, entries=[dict(id="b", tokens=toks[:1], want=[0]), dict(id="a", tokens=toks[29:], want=[0])], end=["a", "b"])]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens",
                        "128", "--device", "cpu"], input="".join(json.dumps(l) + "\n" for l in lines), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    want = O.forward(cfg, w, toks)[0]
    read = lambda n: torch.frombuffer(bytearray((tmp_path / n).read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
    assert M.error(read("0.f32"), want[[3, 19]]) < TOL
    assert M.error(read("2.f32"), torch.stack([want[0], want[29]])) < TOL


def test_random_weights_without_a_checkpoint():
    llm = LLM(hf_config=M.CONFIGS["mixed"], dtype="float32", device="cpu", max_model_len=64)
    o = llm.generate([{"prompt_token_ids": [1, 2, 3]}], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True, detokenize=False))
    assert len(o[0].outputs[0].token_ids) == 4


# ------------------------------------------------------------------------------------------------ what the comparisons would catch
def _mutate(cfg, w, what):
    import copy
    cfg, w = copy.deepcopy(cfg), {k: v.clone() for k, v in w.items()}
    for i, l in enumerate(cfg["layers"]):
        m = l["mixer"]
        if what == "window":
            m["mask"]["size"] += 1
        elif what == "keep":
            m["mask"]["keep_first"] += 1
        elif what == "scale":
            m["scale"] *= 1.02
        elif what == "bias_max":
            m["bias_max"] += 7
        elif what in ("sink", "rel", "g"):
            w[f"l{i}.mix.{what}"].add_(0.25)
        elif what == "ls1":
            w[f"l{i}.ls1"].mul_(1.05)
    if what == "times":
        cfg["loop"]["times"] -= 1
    elif what == "step":
        w["loop.step"] = w["loop.step"].flip(0)
    elif what == "eps":
        cfg["norm"]["eps"] *= 100
    return cfg, w


@pytest.mark.parametrize("what", ["window", "keep", "scale", "bias_max", "sink", "rel", "g", "ls1", "times", "step", "eps"])
def test_mistakes_show_in_the_logits(models, what):
    """A mistake in the restatement (a window or the kept tokens one token off, a shifted sink, a lost pass, ...) moves the logits by far
    more than the tolerance, so the comparisons above would find the same mistake in the engine."""
    cfg, w, _ = models["mixed"]
    toks = M.tokens(cfg, 110, 7)
    assert M.error(O.forward(*_mutate(cfg, w, what), toks)[0], O.forward(cfg, w, toks)[0]) > (5 if what == "eps" else 50) * TOL


def test_ngram_drafts_keep_the_tokens(models):
    cfg, w, path = models["plain"]
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=128, speculative_config=dict(method="ngram", num_speculative_tokens=3))
    p = M.tokens(cfg, 12, 4) * 3
    o = llm.generate([{"prompt_token_ids": p}], SamplingParams(temperature=0.0, max_tokens=30, ignore_eos=True, detokenize=False))
    assert list(o[0].outputs[0].token_ids) == O.greedy(cfg, w, p, 30)


@pytest.mark.timeout(300)
def test_two_tensor_parallel_ranks(tmp_path):
    """Query heads, bias columns, sinks and gates are split over the ranks; keys too, or replicated where a layer has one key head."""
    cfg = M.config(64, 90, [M.layer(4, 2, 16, 24, 3, 64), M.layer(6, 1, 16, 40, 2, 96), M.layer(2, 2, 8, 9, 0, None)], loop=(0, 2, 2))
    w = M.make_weights(cfg, 3, sharp=1.5)
    path = M.save(cfg, w, tmp_path)
    llm = LLM(model=path, dtype="float32", device="cpu", max_model_len=128, tensor_parallel_size=2, distributed_executor_backend="mp")
    prompts = [M.tokens(cfg, n, n) for n in (5, 60)]
    outs = llm.generate([{"prompt_token_ids": p} for p in prompts], SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True, detokenize=False))
    llm.shutdown()
    for p, o in zip(prompts, outs):
        assert list(o.outputs[0].token_ids) == O.greedy(cfg, w, p, 12)


def test_combinations_that_are_not_served_are_refused(models):
    _, _, path = models["plain"]
    for kw in (dict(pipeline_parallel_size=2), dict(kv_cache_dtype="fp8"), dict(tensor_parallel_size=2),
               dict(speculative_config=dict(method="mtp", num_speculative_tokens=1))):
        with pytest.raises(ValueError):
            LLM(model=path, dtype="float32", device="cpu", max_model_len=64, **kw)

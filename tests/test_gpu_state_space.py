"""Mamba-2 models of other families on a B200: the engine's kernels (bf16) against the CPU path (fp32) on the same random checkpoint."""
import pytest
import torch

from gabisun_models import error, replay

pytestmark = pytest.mark.gpu

BAMBA = dict(architectures=["BambaForCausalLM"], hidden_size=256, intermediate_size=192, num_hidden_layers=3, num_attention_heads=4, num_key_value_heads=2, vocab_size=150,
             attn_layer_indices=[1], mamba_n_heads=16, mamba_d_head=32, mamba_d_state=48, mamba_n_groups=2, mamba_d_conv=4, mamba_expand=2, max_position_embeddings=512,
             rms_norm_eps=1e-5, tie_word_embeddings=False)
MAMBA2 = dict(architectures=["Mamba2ForCausalLM"], hidden_size=96, num_hidden_layers=2, num_heads=6, head_dim=32, state_size=40, n_groups=1, expand=2, conv_kernel=3,
              vocab_size=120, time_step_limit=[0.02, 0.4], use_conv_bias=True, layer_norm_epsilon=1e-5, max_position_embeddings=512)


@pytest.mark.parametrize("hf", [BAMBA, MAMBA2], ids=["bamba", "mamba2"])
def test_portions_and_decoding(hf, tmp_path):
    from onecat_vllm.config import ModelConfig
    from onecat_vllm.engine.replay import TraceReplay
    from onecat_vllm.loader.weights import load_model, save_pretrained
    save_pretrained(load_model(ModelConfig.from_hf_dict(dict(hf), dtype=torch.float32, load_format="dummy", seed=3), "cpu"), hf, str(tmp_path))
    g = torch.Generator().manual_seed(0)
    toks = torch.randint(0, hf["vocab_size"], (300,), generator=g).tolist()
    run = TraceReplay(str(tmp_path), "float32", 320, device="cpu")
    want = replay(run, {"a": toks}, [[("a", 300)]])["a"]
    run.close()
    run = TraceReplay(str(tmp_path), "bfloat16", 320, device="cuda")
    for sizes in ([300], [200] + [1] * 100, [64, 2, 3, 130, 1, 100]):
        got = replay(run, {"a": toks}, [[("a", n)] for n in sizes])["a"]
        assert error(got, want) < 0.08, (sizes[:4], error(got, want))
    run.close()

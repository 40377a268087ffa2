"""The engine over a folder with a HuggingFace checkpoint layout (the stage runner's models)."""
import json

import pytest
import torch

pytestmark = pytest.mark.gpu
BF = torch.bfloat16


def _qwen3_folder(path):
    from vexact_b200.checkpoint import write_safetensors

    cfg = dict(model_type="qwen3", num_hidden_layers=2, hidden_size=256, num_attention_heads=4, num_key_value_heads=2,
               head_dim=128, intermediate_size=512, vocab_size=320, rms_norm_eps=1e-6, rope_theta=10000.0,
               torch_dtype="bfloat16")
    g = torch.Generator().manual_seed(0)
    rn = lambda *s: (torch.randn(s, generator=g) * s[-1] ** -0.5).to(BF)   # noqa: E731
    t = {"model.embed_tokens.weight": torch.randn(320, 256, generator=g).to(BF), "model.norm.weight": torch.ones(256, dtype=BF),
         "lm_head.weight": rn(320, 256)}
    for i in range(2):
        p = f"model.layers.{i}."
        t.update({p + "input_layernorm.weight": torch.ones(256, dtype=BF),
                  p + "post_attention_layernorm.weight": torch.ones(256, dtype=BF),
                  p + "self_attn.q_proj.weight": rn(512, 256), p + "self_attn.k_proj.weight": rn(256, 256),
                  p + "self_attn.v_proj.weight": rn(256, 256), p + "self_attn.o_proj.weight": rn(256, 512),
                  p + "self_attn.q_norm.weight": torch.ones(128, dtype=BF),
                  p + "self_attn.k_norm.weight": torch.ones(128, dtype=BF),
                  p + "mlp.gate_proj.weight": rn(512, 256), p + "mlp.up_proj.weight": rn(512, 256),
                  p + "mlp.down_proj.weight": rn(256, 512)})
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(path / "model.safetensors", t)


def test_engine_serves_a_stage_model_folder(tmp_path):
    """Batched, in portions, with and without graphs: the same tokens as each prompt alone."""
    from vexact_b200.engine import Engine
    from vexact_b200.scheduler import GenerationConfig

    _qwen3_folder(tmp_path)
    g = torch.Generator().manual_seed(1)
    prompts = [torch.randint(0, 320, (n,), generator=g).tolist() for n in (40, 5, 17)]
    cfg = GenerationConfig(max_new_tokens=6)
    args = dict(max_num_seqs=4, max_model_len=64, page_size=16)
    alone = Engine.from_folder(tmp_path, max_num_batched_tokens=64, enforce_eager=True, **args)
    want = [alone.generate([p], cfg)[0].generated_tokens for p in prompts]
    for kw in (dict(max_num_batched_tokens=32), dict(max_num_batched_tokens=64, enforce_eager=True)):
        eng = Engine.from_folder(tmp_path, **args, **kw)
        assert [r.generated_tokens for r in eng.generate(prompts, cfg)] == want

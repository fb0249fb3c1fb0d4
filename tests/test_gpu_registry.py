"""GPU: a converted ternary checkpoint folder goes through the registry and the step engine like any other model."""
import json
import sys

import pytest
import torch

pytestmark = pytest.mark.gpu


def fused_state(dim, layers, heads, kv, ffn, vocab):
    g = torch.Generator().manual_seed(0)
    rnd = lambda *s: (torch.randn(s, generator=g) * 0.05).to(torch.bfloat16)
    hd = dim // heads
    out = {"tok_embeddings.weight": rnd(vocab, dim), "norm.weight": 1 + rnd(dim)}
    for i in range(layers):
        p = f"layers.{i}."
        out.update({p + "attention.wqkv.weight": rnd((heads + 2 * kv) * hd, dim), p + "attention.wo.weight": rnd(dim, dim),
                    p + "feed_forward.w13.weight": rnd(2 * ffn, dim), p + "feed_forward.w2.weight": rnd(dim, ffn)})
        out.update({p + n: 1 + rnd(w) for n, w in (("attention.attn_sub_norm.weight", dim), ("feed_forward.ffn_sub_norm.weight", ffn),
                                                   ("attention_norm.weight", dim), ("ffn_norm.weight", dim))})
    return out


def test_converted_folder_is_served(lib, tmp_path, monkeypatch):
    from ternainfer_b200 import registry
    from ternainfer_b200.convert import convert_TernaInfer as conv
    from ternainfer_b200.generate import FastGen, GenArgs, StepEngine
    torch.save(fused_state(256, 2, 2, 1, 384, 500), tmp_path / "in.pt")
    monkeypatch.setattr(sys, "argv", ["convert", "--input", str(tmp_path / "in.pt"), "--output_dir", str(tmp_path), "--dim", "256",
                                      "--n_heads", "2", "--n_kv_heads", "1", "--ffn_dim", "384"])
    conv.main()
    cfg = json.loads((tmp_path / "config.json").read_text())
    assert (cfg["architecture"], cfg["n_layers"], cfg["vocab_size"]) == ("TernaInfer", 2, 500)
    model = registry.load_model(str(tmp_path), torch.bfloat16, 40)
    toks = torch.randint(0, 500, (40,), generator=torch.Generator().manual_seed(1)).tolist()
    with torch.inference_mode():
        want = model(torch.tensor([toks], device="cuda"), model.make_cache(1, "cuda"), torch.arange(40, device="cuda"))[0]
    e = StepEngine(model)
    got = torch.cat([e.step("a", toks[:30], list(range(30))), e.step("a", toks[30:37], list(range(7)))] +
                    [e.step("a", [t], [0]) for t in toks[37:]])
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
    assert err.max() < 0.1          # other token counts use other epilogue forms and attention splits
    prompt = torch.tensor([toks[:30]], device="cuda")
    out, _ = FastGen(model, GenArgs(4, 1, 30, True)).generate(prompt)
    row = want[29]
    assert row.max() - row[out[0, 0]] <= 0.05 * row.abs().max()

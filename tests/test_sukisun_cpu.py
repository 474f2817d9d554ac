"""Host side of the Sukisun family: configuration, loading, registry, batches of the engine, trace replay."""
from pathlib import Path

import pytest
import torch

import plain_sukisun as P
import sukisun_cases as S
from coffin_b200.engine.config import EngineConfig
from coffin_b200.engine.llm_engine import LLMEngine
from coffin_b200.engine.replay import TraceReplayer, pool_blocks
from coffin_b200.engine.sequence import SamplingParams
from coffin_b200.models.sukisun.config import SukisunConfig
from test_zufilorn_cpu import Twin

ROOT = Path(__file__).resolve().parents[1]
SMALL = S.config([S.mamba(2, 8, 8, 1, 2, 1), S.latent(2, 8, 4, 8, 16, 12), S.latent(1, 4, 4, 8, 16, 8, kv_from=1)], width=24, vocab=40, ff=16,
                 no_mlp=(0,))


def test_config_round_trip_and_refusals():
    cfg = SukisunConfig.from_hf(S.ALL)
    assert cfg.layer_types == ("mamba2", "latent_attention") * 2 and cfg.num_hidden_layers == 4
    assert SukisunConfig.from_hf(cfg.to_hf()) == SukisunConfig.from_hf(S.ALL, name="checkpoint")
    assert cfg.to_hf() == S.ALL
    assert cfg.layers[0].ff is None and cfg.layers[3].mixer.kv_from == 1 and cfg.layers[1].mixer.kv_from is None
    bad = [dict(S.mamba(), type="mlstm", mlp=None), dict(S.mamba(), mlp={"kind": "moe", "ff": 8}), dict(S.mamba(5, groups=2), mlp=None),
           dict(S.mamba(5, 8, norm_groups=3, groups=1), mlp=None), dict(S.latent(rot_dims=7), mlp=None), dict(S.latent(kv_from=0), mlp=None)]
    for l in bad:
        with pytest.raises(ValueError):
            SukisunConfig.from_hf(dict(S.ALL, layers=[l]))
    for second in (S.latent(kv_rank=64, kv_from=0), S.latent(base=100.0, kv_from=0), S.latent(rot_dim=8, kv_from=0)):
        with pytest.raises(ValueError):
            SukisunConfig.from_hf(S.config([S.latent(), second]))
    with pytest.raises(ValueError):                                # a layer without latents of its own cannot lend any
        SukisunConfig.from_hf(S.config([S.latent(), S.latent(kv_from=0), S.latent(kv_from=1)]))


def test_tensor_plan_names_what_the_plain_model_reads():
    plan = {n: s for n, s, _ in SukisunConfig.from_hf(S.ALL).tensor_plan()}
    W = S.weights(S.ALL)
    assert plan == {n: tuple(t.shape) for n, t in W.items()}


def test_checkpoint_directory_registry_and_random_weights(tmp_path):
    from coffin_b200.config import load_config, preset
    from coffin_b200.models import FLOAT32, detect_architecture, kernel_sources
    from coffin_b200.weights.init import param_count, random_state_dict, save_checkpoint
    from coffin_b200.weights.loader import load_checkpoint
    cfg = preset("tiny-sukisun")
    sd = random_state_dict(cfg, 1, dtype=torch.bfloat16)
    assert sum(t.numel() for t in sd.values()) == param_count(cfg)
    save_checkpoint(cfg, sd, tmp_path)
    back = load_checkpoint(tmp_path)
    assert set(back) == set(sd) and all(torch.equal(back[k], sd[k]) for k in sd)
    assert detect_architecture(load_config(tmp_path)) == "sukisun" and "sukisun" in FLOAT32
    assert all((ROOT / "coffin_b200" / "_C" / f).exists() for f in kernel_sources("sukisun"))
    lg = P.forward(cfg.to_hf(), {k: v.bfloat16() for k, v in sd.items()}, [1, 2, 3])
    assert lg.shape == (3, cfg.vocab_size) and torch.isfinite(lg).all()
    assert all(preset(n).num_hidden_layers > 8 for n in ("sukisun-1b", "sukisun-4b"))


def test_plain_recurrence_and_attention_ignore_what_comes_later():
    W = S.weights(S.ALL, 1)
    ids = [(7 * k) % 96 for k in range(12)]
    a = P.forward(S.ALL, W, ids, torch.float64)
    assert torch.allclose(a[:7], P.forward(S.ALL, W, ids[:7], torch.float64), atol=1e-9)


def plain_greedy(cfg, W, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(P.forward(cfg, W, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("mixed,blocks", [(True, 16), (True, 5), (False, 5)])
def test_engine_steps_mix_prompts_and_decode_rows(mixed, blocks):
    """Same greedy tokens with and without mixed steps, also on a pool that preempts."""
    W = S.weights(SMALL, 2)
    twin = Twin(SMALL, W, slots=3, blocks=blocks, forward=P.forward)
    eng = LLMEngine(twin, EngineConfig(max_seq=256, max_num_seqs=3, chunk=24, prefill_quantum=24, max_num_batched_tokens=40,
                                       mixed_batch=mixed, prefix_cache=False))
    prompts = [[(7 * i + k) % 40 for k in range(n)] for i, n in enumerate((60, 5, 70, 30))]
    seqs = eng.generate(prompts, SamplingParams(max_tokens=5, ignore_eos=True))
    assert [s.output for s in seqs] == [plain_greedy(SMALL, W, p, 5) for p in prompts]
    assert bool([b for b in twin.batches if max(b) > 1 and min(b) == 1]) == mixed and eng.bm.pool.used_blocks == 0


def test_trace_replay_batches_admission_and_release():
    W = S.weights(SMALL, 3)
    twin = Twin(SMALL, W, slots=4, blocks=pool_blocks(192), forward=P.forward)
    rep = TraceReplayer(twin)
    a, b = ([(3 * k + i) % 40 for k in range(n)] for i, n in enumerate((100, 64)))
    out = rep.step([{"id": "a", "tokens": a[:70], "want": [0, 69]}, {"id": "b", "tokens": b[:1], "want": []}])
    ref = {k: P.forward(SMALL, W, v) for k, v in (("a", a), ("b", b))}
    assert torch.allclose(out, ref["a"][[0, 69]], atol=1e-4) and twin.batches == [[70, 1]]
    assert rep.step([{"id": "b", "tokens": b[1:63], "want": []}]) is None            # a sits out
    out = rep.step([{"id": "b", "tokens": b[63:], "want": [0]}, {"id": "a", "tokens": a[70:71], "want": [0]}], ["b"])
    assert torch.allclose(out, torch.stack([ref["b"][63], ref["a"][70]]), atol=1e-4)
    rep.engine.reset()

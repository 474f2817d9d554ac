"""Host side of the Zufilorn family: configuration, loading, registry, batches of the engine, trace replay."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_zufilorn as P
import zufilorn_cases as Z
from coffin_b200.engine.config import EngineConfig
from coffin_b200.engine.llm_engine import LLMEngine
from coffin_b200.engine.replay import TraceReplayer, pool_blocks
from coffin_b200.engine.sequence import SamplingParams
from coffin_b200.models.zufilorn.config import ZufilornConfig

ROOT = Path(__file__).resolve().parents[1]


class Twin:
    """The model interface of the engine on the CPU: a slot holds the tokens it was fed, logits come from the plain
    model run over all of them.  Positions and tables are checked, so a batch the engine builds wrongly fails."""
    mixed_batches = True

    def __init__(self, cfg, W, slots, blocks, max_seq=256, forward=P.forward):
        self.cfg_raw, self.W, self.device, self.forward = cfg, W, torch.device("cpu"), forward
        self.num_slots, self.num_blocks, self.max_seq, self.max_chunk = slots, blocks, max_seq, 2048
        self.fed = [[] for _ in range(slots)]
        self.batches = []

    def zero_state(self, slot):
        self.fed[slot] = []

    def snapshot_state(self, slot):
        return list(self.fed[slot])

    def restore_state(self, slot, snap):
        self.fed[slot] = list(snap)

    def copy_block(self, src, dst):
        pass

    def sample(self, logits, temps, us):
        return logits.argmax(-1)

    def forward_batch(self, items, want):
        self.batches.append([len(t) for t, *_ in items])
        assert len({s for _t, _p, s, _b in items}) == len(items)
        rows = []
        for (toks, pos0, slot, table), w in zip(items, want):
            toks = toks.tolist() if isinstance(toks, torch.Tensor) else list(toks)
            assert pos0 == len(self.fed[slot]) and len(table) * 64 >= pos0 + len(toks) and 0 not in table
            self.fed[slot] += toks
            if w:
                lg = self.forward(self.cfg_raw, self.W, self.fed[slot])
                rows += [lg[pos0 + i] for i in w]
        return torch.stack(rows) if rows else None

    def prefill(self, tokens, pos0, slot, table, embeds=None, cos_sin=None, want_logits=True):
        out = self.forward_batch([(tokens, pos0, slot, table)], [[len(tokens) - 1] if want_logits else []])
        return out[0] if want_logits else None

    @staticmethod
    def bucket_for(n):
        return n

    def set_rows(self, M, tokens, positions, slots, tables, deltas=None):
        self.rows = [([t], p, s, b) for t, p, s, b in zip(tokens, positions, slots, tables)]

    def decode(self, M, graph=True):
        lg = self.forward_batch(self.rows, [[0]] * len(self.rows))
        return lg.argmax(-1), lg


SMALL = Z.config([Z.mlstm(2, 8, 8), Z.attention(2, 1, 8, 8)], width=24, vocab=40, ff=16, max_positions=300)


def test_config_round_trip_and_refusals():
    cfg = ZufilornConfig.from_hf(Z.ALL)
    assert cfg.layer_types == ("channel_delta", "mlstm", "attention") and cfg.num_hidden_layers == 3
    assert ZufilornConfig.from_hf(cfg.to_hf()) == ZufilornConfig.from_hf(Z.ALL, name="checkpoint")
    none = Z.config([Z.attention(softcap=None, every=0)], no_mlp=(0,))
    c = ZufilornConfig.from_hf(none)
    assert c.layers[0].ff is None and c.layers[0].mixer.softcap is None and c.layers[0].mixer.temp_every == 0
    for bad in ({"type": "mamba", "mixer": {}, "mlp": None}, dict(Z.mlstm(), mlp={"kind": "moe", "ff": 8})):
        with pytest.raises(ValueError):
            ZufilornConfig.from_hf(dict(Z.ALL, layers=[bad]))
    with pytest.raises(ValueError):
        ZufilornConfig.from_hf(dict(Z.ALL, layers=[dict(Z.delta(3, 2), mlp=None)]))


def test_tensor_plan_names_what_the_plain_model_reads():
    plan = {n: s for n, s, _ in ZufilornConfig.from_hf(Z.ALL).tensor_plan()}
    W = Z.weights(Z.ALL, rank=24)
    assert set(plan) == set(W)
    low = ("a1", "a2", "g1", "g2")
    assert all(plan[n] == tuple(t.shape) for n, t in W.items() if n.rpartition(".")[2] not in low)


def test_checkpoint_directory_registry_and_random_weights(tmp_path):
    from coffin_b200.config import load_config, preset
    from coffin_b200.models import detect_architecture, kernel_sources
    from coffin_b200.weights.init import param_count, random_state_dict, save_checkpoint
    from coffin_b200.weights.loader import load_checkpoint
    cfg = preset("tiny-zufilorn")
    sd = random_state_dict(cfg, 1, dtype=torch.bfloat16)
    assert sum(t.numel() for t in sd.values()) == param_count(cfg)
    save_checkpoint(cfg, sd, tmp_path)
    back = load_checkpoint(tmp_path)
    assert set(back) == set(sd) and all(torch.equal(back[k], sd[k]) for k in sd)
    assert detect_architecture(load_config(tmp_path)) == "zufilorn"
    assert all((ROOT / "coffin_b200" / "_C" / f).exists() for f in kernel_sources("zufilorn"))
    lg = P.forward(cfg.to_hf(), sd, [1, 2, 3])
    assert lg.shape == (3, cfg.vocab_size) and torch.isfinite(lg).all()
    assert all(preset(n).num_hidden_layers > 8 for n in ("zufilorn-1b", "zufilorn-4b"))


def plain_greedy(cfg, W, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(P.forward(cfg, W, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("mixed", [True, False])
@pytest.mark.parametrize("blocks", [16, 5])
def test_engine_steps_mix_prompts_and_decode_rows(mixed, blocks):
    """Same greedy tokens with and without mixed steps, also on a pool that preempts."""
    W = Z.weights(SMALL, 2)
    twin = Twin(SMALL, W, slots=3, blocks=blocks)
    eng = LLMEngine(twin, EngineConfig(max_seq=256, max_num_seqs=3, chunk=24, prefill_quantum=24, max_num_batched_tokens=40,
                                       mixed_batch=mixed, prefix_cache=False))
    prompts = [[(7 * i + k) % 40 for k in range(n)] for i, n in enumerate((60, 5, 70, 30))]
    seqs = eng.generate(prompts, SamplingParams(max_tokens=7, ignore_eos=True))
    assert [s.output for s in seqs] == [plain_greedy(SMALL, W, p, 7) for p in prompts]
    both = [b for b in twin.batches if max(b) > 1 and min(b) == 1]
    assert bool(both) == mixed and eng.bm.pool.used_blocks == 0
    assert all(sum(b) <= 40 for b in twin.batches)


def test_trace_replay_batches_admission_and_release():
    W = Z.weights(SMALL, 3)
    twin = Twin(SMALL, W, slots=4, blocks=pool_blocks(192))
    rep = TraceReplayer(twin)
    a, b, c = ([(3 * k + i) % 40 for k in range(n)] for i, n in enumerate((100, 64, 20)))
    out = rep.step([{"id": "a", "tokens": a[:70], "want": [0, 69]}, {"id": "b", "tokens": b[:1], "want": []}])
    ref = {k: P.forward(SMALL, W, v) for k, v in (("a", a), ("b", b), ("c", c))}
    assert torch.allclose(out, ref["a"][[0, 69]], atol=1e-4) and twin.batches == [[70, 1]]
    assert rep.step([{"id": "b", "tokens": b[1:63], "want": []}]) is None            # a sits out
    out = rep.step([{"id": "b", "tokens": b[63:], "want": [0]}, {"id": "a", "tokens": a[70:71], "want": [0]}], ["b"])
    assert torch.allclose(out, torch.stack([ref["b"][63], ref["a"][70]]), atol=1e-4)
    with pytest.raises(RuntimeError):                                                # the pool holds three pages
        rep.step([{"id": "d", "tokens": [1] * 80, "want": []}])
    rep.engine.reset()


def test_models_without_mixed_batches_replay_entry_by_entry():
    """The Qwen3.5 CPU twin has no mixed forward: portions are cut at the wanted places."""
    from coffin_b200.config import ModelConfig
    from coffin_b200.oracle.engine_model import OracleEngineModel
    from coffin_b200.weights.init import random_state_dict
    cfg = ModelConfig(vocab_size=64, hidden_size=32, num_hidden_layers=2, layer_types=("linear_attention", "full_attention"),
                      num_attention_heads=2, num_key_value_heads=1, head_dim=16, linear_num_key_heads=2, linear_num_value_heads=2,
                      linear_key_head_dim=16, linear_value_head_dim=16, intermediate_size=48, mrope_section=(3, 3, 2), partial_rotary_factor=1.0)
    sd = random_state_dict(cfg, 4)
    ids = [(5 * k) % 64 for k in range(30)]
    one = TraceReplayer(OracleEngineModel(cfg, sd, max_seq=128, num_slots=4))
    whole = one.step([{"id": "x", "tokens": ids, "want": [4, 20, 29]}], ["x"])
    two = TraceReplayer(OracleEngineModel(cfg, sd, max_seq=128, num_slots=4))
    got = [two.step([{"id": "x", "tokens": ids[:12], "want": [4]}, {"id": "y", "tokens": ids[:3], "want": []}]),
           two.step([{"id": "x", "tokens": ids[12:29], "want": [8]}]), two.step([{"id": "x", "tokens": ids[29:], "want": [0]}])]
    assert torch.allclose(torch.cat(got), whole, atol=1e-4)


def test_trace_run_program_refuses_a_16_bit_family_in_32_bit(tmp_path):
    from coffin_b200.config import ModelConfig
    (tmp_path / "config.json").write_text(json.dumps(ModelConfig().to_hf()))
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "64"], capture_output=True, text=True, input="")
    assert r.returncode == 3 and "16 bits" in r.stderr

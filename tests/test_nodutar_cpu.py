"""Host side of the Nodutar family: configuration, loading, registry, weight layouts, batches of the engine, trace replay."""
import copy
from pathlib import Path

import pytest
import torch

import nodutar_cases as S
import plain_nodutar as P
from coffin_b200.engine.config import EngineConfig
from coffin_b200.engine.llm_engine import LLMEngine
from coffin_b200.engine.replay import TraceReplayer, pool_blocks
from coffin_b200.engine.sequence import SamplingParams
from coffin_b200.models.nodutar.config import Loop, NodutarConfig, RoutedFF
from test_zufilorn_cpu import Twin

ROOT = Path(__file__).resolve().parents[1]
SMALL = S.config([S.parallel(2, 1, 8, 8, 20, 4, mem=(2, 4, 4)), S.attention(2, 1, 8)], [S.moe(3, 2, 8), None], (0, 2, 2), width=24, vocab=40)


def test_config_round_trip_and_refusals():
    cfg = NodutarConfig.from_hf(S.ALL)
    assert cfg.layer_types == ("attention", "parallel", "attention", "parallel", "parallel") and cfg.loop == Loop(1, 3, 3)
    assert NodutarConfig.from_hf(cfg.to_hf()) == NodutarConfig.from_hf(S.ALL, name="checkpoint")
    assert cfg.to_hf() == S.ALL and NodutarConfig.from_hf(SMALL).to_hf() == SMALL
    assert cfg.layers[2].ff is None and cfg.layers[1].ff == RoutedFF(24, 5, 2) and cfg.layers[4].mixer.left.chunk == 70
    one = lambda l, f=None, loop=None: S.config([l], [f], loop)
    bad = [one(dict(S.attention(), type="mamba2")), one(S.attention(5, 2)), one(S.parallel(5, 2)), one(S.parallel(rot=7)), one(S.parallel(rot=26)), one(S.parallel(vdim=7)),
           one(S.attention(), {"kind": "glu", "ff": 8}), one(S.attention(), S.moe(top=8)), one(S.attention(), S.moe(513, 1)), one(S.attention(), S.moe(40, 33)),
           one(S.attention(), None, (0, 2, 2)), one(S.attention(), None, (0, 1, 0)), one(S.attention(), None, (1, 1, 2)),
           one(dict(S.attention(), mixer=dict(S.attention()["mixer"], vdim=48)))]
    broken = copy.deepcopy(one(S.parallel()))
    broken["layers"][0]["mixer"]["left"]["mask"] = {"size": 0}
    for raw in bad + [broken]:
        with pytest.raises(ValueError):
            NodutarConfig.from_hf(raw)


def test_optional_parts_of_the_configuration():
    raw = copy.deepcopy(S.config([S.parallel()], [None]))
    del raw["loop"], raw["layers"][0]["mixer"]["left"]["mask"], raw["layers"][0]["mlp"]
    cfg = NodutarConfig.from_hf(raw)
    assert cfg.loop is None and cfg.layers[0].ff is None and cfg.layers[0].mixer.left.chunk == 0 and cfg.runs() == [(0, 0, False)]


@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 5, 2), (1, 3, 3), (4, 5, 2), (2, 5, 1)])
def test_order_of_runs(loop):
    raw = dict(S.ALL, loop=dict(zip(("start", "stop", "times"), loop)) if loop else None)
    runs = NodutarConfig.from_hf(raw).runs()
    assert [(i, a) for i, _, a in runs] == P.run_order(raw)
    assert len(set((i, k) for i, k, _ in runs)) == len(runs) and {i for i, _, _ in runs} == set(range(5))
    cut = NodutarConfig.from_hf(raw).first_layers(3)
    assert cut.num_hidden_layers == 3 and (cut.loop is None) == (not loop or loop[1] > 3)


@pytest.mark.parametrize("raw", [S.ALL, SMALL])
def test_tensor_plan_names_what_the_plain_model_reads(raw):
    plan = {n: s for n, s, _ in NodutarConfig.from_hf(raw).tensor_plan()}
    assert plan == {n: tuple(t.shape) for n, t in S.weights(raw).items()}


def test_checkpoint_directory_registry_and_random_weights(tmp_path):
    from coffin_b200.config import load_config, preset
    from coffin_b200.models import FLOAT32, detect_architecture, kernel_sources, registered
    from coffin_b200.weights.init import param_count, random_state_dict, save_checkpoint
    from coffin_b200.weights.loader import load_checkpoint
    cfg = preset("tiny-nodutar")
    sd = random_state_dict(cfg, 1, dtype=torch.bfloat16)
    assert sum(t.numel() for t in sd.values()) == param_count(cfg)
    save_checkpoint(cfg, sd, tmp_path)
    back = load_checkpoint(tmp_path)
    assert set(back) == set(sd) and all(torch.equal(back[k], sd[k]) for k in sd)
    assert detect_architecture(load_config(tmp_path)) == "nodutar" and "nodutar" in FLOAT32 and "nodutar" in registered()
    assert all((ROOT / "coffin_b200" / "_C" / f).exists() for f in kernel_sources("nodutar"))
    lg = P.forward(cfg.to_hf(), {k: v.bfloat16() for k, v in sd.items()}, [1, 2, 3])
    assert lg.shape == (3, cfg.vocab_size) and torch.isfinite(lg).all()
    assert [len(preset(n).runs()) for n in ("nodutar-35b-a3b", "nodutar-3b")] == [40, 20]


def test_gated_experts_keep_gate_rows_before_up_rows():
    from coffin_b200.models.experts import RoutedExperts
    g = torch.Generator().manual_seed(2)
    W = {f"e{e}.{n}": torch.randn(s, generator=g) for e in range(3) for n, s in (("gate", (13, 20)), ("up", (13, 20)), ("down", (20, 13)))}
    W |= {"router": torch.randn(3, 20, generator=g), "router.b": torch.zeros(3)}
    W |= {"shared.gate": torch.randn(17, 20, generator=g), "shared.up": torch.randn(17, 20, generator=g), "shared.down": torch.randn(20, 17, generator=g)}
    r = RoutedExperts(W, experts=3, top=2, ff=13, shared=17, width=20, dtype=torch.float32, dev="cpu", gated=True, by_logit=True, correction="router.b")
    h = torch.zeros(4, 24)
    h[:, :20] = torch.randn(4, 20, generator=g)
    one = lambda e: (P.silu(h @ r.up[e, :16].T) * (h @ r.up[e, 16:].T)) @ r.down[e].T
    plain = lambda n: (P.silu(h[:, :20] @ W[n + "gate"].T) * (h[:, :20] @ W[n + "up"].T)) @ W[n + "down"].T
    assert r.r.by_logit and r.r.always == 2 and r.up.shape == (5, 32, 24)
    assert all(torch.allclose(one(e)[:, :20], plain(f"e{e}."), atol=1e-4) for e in range(3))
    assert torch.allclose((one(3) + one(4))[:, :20], plain("shared."), atol=1e-4)


def test_runs_of_a_layer_share_weights_but_not_pages_or_state(monkeypatch):
    from coffin_b200.models.nodutar import mixers as M
    made = []
    monkeypatch.setattr(M.X, "AttnMaps", lambda **kw: made.append(kw))
    monkeypatch.setattr(M.X, "Linrec", lambda kind, **kw: made.append(kw))
    cfg, W = NodutarConfig.from_hf(S.ALL), S.weights(S.ALL)
    mix = lambda i: {k[len(f"l{i}.mix."):]: v for k, v in W.items() if k.startswith(f"l{i}.mix.")}
    a = M.Parallel(cfg.layers[1].mixer, mix(1), 72, 1e-5, 3, 2, torch.float32, "cpu")
    b = a.twin()
    assert b.w_out is a.w_out and b.proj is a.proj and b.state["S"] is not a.state["S"] and all(p is not q for p, q in zip(a.pools, b.pools))
    assert torch.allclose(a.gates["norm_w"], W["l1.mix.right.norm"].float() * 1.6) and made[0]["chunk"] == 50 and made[0]["out_scale"] == 0.7
    assert made[2]["kpool"] is b.pools[0] and made[3]["state"] is b.state and made[1]["lower"] is made[3]["lower"]
    c = M.DistanceAttention(cfg.layers[0].mixer, mix(0), 72, 1e-5, 3, torch.float32, "cpu")
    d = c.twin()
    assert [tuple(p.shape) for p in c.pools] == [(192, 2, 40), (192, 2)] and c.pools[1].dtype == torch.float32
    assert made[5]["factors"] is d.pools[1] is not c.pools[1] and not c.state


def test_bound_of_scores():
    from coffin_b200.ops.mixers import MAX_BOUND, AttnMaps
    one, two, r = torch.ones(16), torch.full((16,), -2.0), torch.tensor([0.5, 0.0])
    assert AttnMaps._bound(0.25, 16, None, None) == 0 and AttnMaps._bound(0.25, 16, (1e-6, None, None), None) == pytest.approx(4.08)
    assert AttnMaps._bound(-0.25, 16, (1e-6, two, one), (r, r)) == pytest.approx(8.16)
    assert AttnMaps._bound(0.25, 16, (1e-6, None, None), (r, -r)) == 0 and AttnMaps._bound(MAX_BOUND / 16, 16, (1e-6, None, None), None) == 0


def test_splits_cover_the_pages_of_a_chunk():
    from coffin_b200.ops.mixers import window_pages
    for size in (1, 2, 63, 64, 65, 66, 128, 130, 1000):
        assert max(p // 64 - p // size * size // 64 + 1 for p in range(5 * size * 64)[:20000]) <= window_pages(size)


def test_plain_model_ignores_what_comes_later_and_other_chunks():
    W = S.weights(S.ALL, 1)
    ids = [(7 * k) % 96 for k in range(12)]
    a = P.forward(S.ALL, W, ids, torch.float64)
    assert torch.allclose(a[:7], P.forward(S.ALL, W, ids[:7], torch.float64), atol=1e-9)
    h, m = torch.randn(12, 72, dtype=torch.float64), dict(S.parallel(chunk=5)["mixer"]["left"])
    w = {k[len("l1.mix.left."):]: v.double() for k, v in W.items() if k.startswith("l1.mix.left.")}
    other = h.clone()
    other[3] += 1.0
    x, y = P.chunk_attention(h, w, m, 1e-5), P.chunk_attention(other, w, m, 1e-5)
    assert torch.allclose(x[5:], y[5:]) and torch.allclose(x[:3], y[:3]) and not torch.allclose(x[4], y[4])


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

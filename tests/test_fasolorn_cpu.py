"""Host side of the Fasolorn family: configuration, loading, registry, weight layouts, batches of the engine, trace replay."""
import copy
from pathlib import Path

import pytest
import torch

import fasolorn_cases as S
import plain_fasolorn as P
from coffin_b200.engine.config import EngineConfig
from coffin_b200.engine.llm_engine import LLMEngine
from coffin_b200.engine.replay import TraceReplayer, pool_blocks
from coffin_b200.engine.sequence import SamplingParams
from coffin_b200.models.fasolorn.config import FasolornConfig, RoutedFF
from test_zufilorn_cpu import Twin

ROOT = Path(__file__).resolve().parents[1]
SMALL = S.config([S.attention(2, 1, 8, 8, 20, 4), S.latent(2, 8, 4, 8, 16, 30), S.attention(1, 1, 4, 8, 0, 2, v_mix=False)],
                 [S.dense(16), S.moe(3, 1, 2, 8, 12), None], width=24, vocab=40)


def test_config_round_trip_and_refusals():
    cfg = FasolornConfig.from_hf(S.ALL)
    assert cfg.layer_types == ("attention", "latent_attention", "attention", "attention", "latent_attention")
    assert FasolornConfig.from_hf(cfg.to_hf()) == FasolornConfig.from_hf(S.ALL, name="checkpoint")
    assert cfg.to_hf() == S.ALL and FasolornConfig.from_hf(SMALL).to_hf() == SMALL
    assert cfg.first_mixed == 0 and cfg.layers[3].ff is None and cfg.layers[1].ff == RoutedFF(40, 7, 3, 3, 1.5, 56)
    assert FasolornConfig.from_hf(SMALL).layers[2].mixer.window == 0
    one = lambda l, f=None: S.config([l], [f])
    bad = [one(dict(S.attention(), type="mamba2")), one(S.attention(5, 2)), one(S.attention(rot=7)), one(S.attention(rot=26)), one(S.latent(), {"kind": "glu", "ff": 8}),
           one(S.latent(), S.moe(top=11)), one(S.latent(), S.moe(experts=500, identity=13)), one(S.latent(), S.moe(40, top=33)),
           one(dict(S.attention(), mixer=dict(S.attention()["mixer"], mask={"size": 0}))),
           S.config([S.attention(), S.attention(6, 3)], [None, None])]
    for raw in bad:
        with pytest.raises(ValueError):
            FasolornConfig.from_hf(raw)
    FasolornConfig.from_hf(S.config([S.attention(6, 3, v_mix=False), S.attention(), S.attention(4, 1, vdim=80)], [None] * 3))


def test_optional_parts_of_the_configuration():
    raw = copy.deepcopy(S.config([S.latent()], [S.moe(4, 0, 2, 16, 0)]))
    del raw["layers"][0]["mlp"]["router"]["identity"], raw["layers"][0]["mlp"]["shared"], raw["layers"][0]["mixer"]["mask"]
    cfg = FasolornConfig.from_hf(raw)
    assert cfg.layers[0].ff == RoutedFF(16, 4, 0, 2, 1.5, 0) and cfg.layers[0].mixer.window == 0 and cfg.first_mixed is None


@pytest.mark.parametrize("raw", [S.ALL, SMALL])
def test_tensor_plan_names_what_the_plain_model_reads(raw):
    plan = {n: s for n, s, _ in FasolornConfig.from_hf(raw).tensor_plan()}
    assert plan == {n: tuple(t.shape) for n, t in S.weights(raw).items()}


def test_checkpoint_directory_registry_and_random_weights(tmp_path):
    from coffin_b200.config import load_config, preset
    from coffin_b200.models import FLOAT32, detect_architecture, kernel_sources
    from coffin_b200.weights.init import param_count, random_state_dict, save_checkpoint
    from coffin_b200.weights.loader import load_checkpoint
    cfg = preset("tiny-fasolorn")
    sd = random_state_dict(cfg, 1, dtype=torch.bfloat16)
    assert sum(t.numel() for t in sd.values()) == param_count(cfg)
    save_checkpoint(cfg, sd, tmp_path)
    back = load_checkpoint(tmp_path)
    assert set(back) == set(sd) and all(torch.equal(back[k], sd[k]) for k in sd)
    assert detect_architecture(load_config(tmp_path)) == "fasolorn" and "fasolorn" in FLOAT32
    assert all((ROOT / "coffin_b200" / "_C" / f).exists() for f in kernel_sources("fasolorn"))
    lg = P.forward(cfg.to_hf(), {k: v.bfloat16() for k, v in sd.items()}, [1, 2, 3])
    assert lg.shape == (3, cfg.vocab_size) and torch.isfinite(lg).all()
    assert all(preset(n).num_hidden_layers > 8 for n in ("fasolorn-4b", "fasolorn-35b-a3b"))


def test_reordered_rows_turn_like_halves():
    """Rows of a half-paired rotation, reordered at load, give the same scores when neighbours turn."""
    from coffin_b200.models.latent import halves_to_pairs
    g = torch.Generator().manual_seed(1)
    for n, dims in ((16, 16), (12, 8), (6, 2), (10, 10)):
        wq, wk, h = (torch.randn(s, generator=g, dtype=torch.float64) for s in ((n, 20), (n, 20), (9, 20)))
        a = P.rotate_halves(h @ wq.T, dims, 40.0) @ P.rotate_halves(h @ wk.T, dims, 40.0).T
        b = P.rotate_pairs(h @ halves_to_pairs(wq, dims).T, dims, 40.0) @ P.rotate_pairs(h @ halves_to_pairs(wk, dims).T, dims, 40.0).T
        assert torch.allclose(a, b, atol=1e-10)
        assert not torch.allclose(a, P.rotate_pairs(h @ wq.T, dims, 40.0) @ P.rotate_pairs(h @ wk.T, dims, 40.0).T) or dims == 2


def test_shared_expert_in_parts_is_the_whole():
    from coffin_b200.models.experts import RoutedExperts
    for ff, shared in ((40, 56), (24, 24), (16, 70), (32, 8), (24, 0), (4, 300), (1, 20), (1, 16), (2, 33)):
        mlp = S.moe(3, 1, 2, ff, shared)
        W = {k[7:]: v for k, v in S.weights(S.config([S.latent()], [mlp])).items() if k.startswith("l0.mlp.")}
        r = RoutedExperts(W, experts=3, identity=1, top=2, scale=1.5, ff=ff, shared=shared, width=72, dtype=torch.float32, dev="cpu")
        assert r.r.always == -(-shared // max(ff, -(-shared // 16))) and r.r.slots == 2 + r.r.always <= 18
        h = torch.randn(5, 72)
        got = sum((torch.relu(h @ r.up[3 + p].T) ** 2 @ r.down[3 + p].T for p in range(r.r.always)), torch.zeros(5, 72))
        ref = P.squared_relu(h, W["shared.up"].float(), W["shared.down"].float()) if shared else torch.zeros(5, 72)
        assert torch.allclose(got, ref, atol=1e-4)


def test_pages_of_a_window():
    from coffin_b200.models.rowmodel import RowBatch
    from coffin_b200.ops.mixers import window_pages
    for win in (1, 2, 63, 64, 65, 66, 128, 129, 130, 1000):
        seen = max(p // 64 - max(0, p - win + 1) // 64 + 1 for p in range(3000))
        assert window_pages(win) == seen
    assert window_pages(0) > 10 ** 6
    z = torch.zeros(1, dtype=torch.int32)
    b = RowBatch(T=200, n_seg=2, n_pre=2, pre_rows=200, tokens=z, positions=z, row_seg=None, seg_row=None, seg_pos=z, seg_slot=z, tables=z,
                 pre_lens=(400, 170), pre_pos=(300, 70))
    for win, skip in ((0, (0, 0)), (60, (3, 0)), (43, (4, 0)), (46, (3, 0)), (45, (4, 0)), (7, (4, 1)), (1, (4, 1))):
        e = b.expansion(win)
        assert tuple(e["skip"].tolist()) == skip and e["lens"].tolist() == [400 - 64 * skip[0], 170 - 64 * skip[1]], win
        assert e["pos"].tolist() == [300 - 64 * skip[0], 70 - 64 * skip[1]]
        pages = [-(-n // 64) for n in e["lens"].tolist()]
        assert e["rows"] == 64 * sum(pages) and e["base"].tolist() == [0, 64 * pages[0]] and e["pages"] == max(pages)
        assert e["tables"][1, :pages[1]].tolist() == list(range(pages[0], sum(pages)))
    assert b.expansion(60) is b.expansion(60)


def test_plain_model_ignores_what_comes_later_and_what_left_the_window():
    W = S.weights(S.ALL, 1)
    ids = [(7 * k) % 96 for k in range(12)]
    a = P.forward(S.ALL, W, ids, torch.float64)
    assert torch.allclose(a[:7], P.forward(S.ALL, W, ids[:7], torch.float64), atol=1e-9)
    one = S.config([S.attention(window=5)], [None])
    W = S.weights(one, 1)
    a, b = (P.forward(one, W, x, torch.float64) for x in (ids, [3] + ids[1:]))
    assert torch.allclose(a[5:], b[5:]) and not torch.allclose(a[4], b[4])


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


class PagedTwin(Twin):
    """The twin of a model whose pages are all the state: what a sequence was fed is read back through its block table."""
    stateless = True

    def __init__(self, *a, **kw):
        super().__init__(*a, **kw)
        self.pages = [[None] * 64 for _ in range(self.num_blocks)]

    def forward_batch(self, items, want):
        for toks, pos0, slot, table in items:
            self.fed[slot] = [self.pages[table[i // 64]][i % 64] for i in range(pos0)]
            for i, t in enumerate(toks.tolist() if isinstance(toks, torch.Tensor) else toks):
                self.pages[table[(pos0 + i) // 64]][(pos0 + i) % 64] = t
        return super().forward_batch(items, want)

    def copy_block(self, src, dst):
        self.pages[dst] = list(self.pages[src])

    def snapshot_state(self, slot):
        raise AssertionError("nothing to take a snapshot of")

    restore_state = snapshot_state


def test_any_cached_page_prefix_is_reused_without_snapshots():
    W = S.weights(SMALL, 4)
    twin = PagedTwin(SMALL, W, slots=2, blocks=24, forward=P.forward)
    eng = LLMEngine(twin, EngineConfig(max_seq=256, max_num_seqs=2, chunk=100, prefill_quantum=100, mixed_batch=True))
    base = [(5 * k) % 40 for k in range(180)]
    prompts = [base, base[:70] + [1, 2, 3], base[:150] + [9] * 20, base[:64] + [4]]
    params = SamplingParams(max_tokens=4, ignore_eos=True)
    cached = 0
    for p, n in zip(prompts, (0, 64, 128, 64)):
        s, = eng.generate([p], params)
        assert s.output == plain_greedy(SMALL, W, p, 4)
        assert eng.runner.n_cached_tokens - cached == n
        cached = eng.runner.n_cached_tokens
    assert any(100 in b for b in twin.batches)                     # no chunk was cut for a snapshot's sake


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

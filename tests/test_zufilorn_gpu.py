"""Zufilorn on the device against the plain restatement of its equations (``plain_zufilorn.py``)."""
import random

import pytest
import torch

import plain_zufilorn as P
import zufilorn_cases as Z

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
# rms of the error over the rms of the value: 32-bit mode, serving mode
TOL = {F32: 2e-5, BF16: 3e-2}


def build(cfg, W, dtype=F32, slots=4, blocks=40, max_seq=640, **kw):
    from coffin_b200.models import build_model
    from coffin_b200.models.zufilorn.config import ZufilornConfig
    c = ZufilornConfig.from_hf(cfg)
    return build_model(c, W, device="cuda", dtype=dtype, num_slots=slots, num_blocks=blocks, max_seq=max_seq, **kw)


def rel(got, ref):
    got, ref = got.double().cpu(), ref.double().cpu()
    return float((got - ref).pow(2).mean().sqrt() / ref.pow(2).mean().sqrt().clamp_min(1e-30))


def toks(n, vocab, seed=0):
    r = random.Random(seed)
    return [r.randrange(vocab) for _ in range(n)]


def table(n, first=1, step=1):
    return [first + step * i for i in range((n + 63) // 64)]


def run_portions(m, ids, cuts, slot=0, tab=None, want_all=True):
    """Logits of every position, the sequence cut into portions of the given sizes (cycled)."""
    tab = tab or table(len(ids))
    m.zero_state(slot)
    out, at, k = [], 0, 0
    while at < len(ids):
        n = min(cuts[k % len(cuts)], len(ids) - at)
        k += 1
        out.append(m.forward_batch([(ids[at:at + n], at, slot, tab)], [list(range(n))]).clone())
        at += n
    return torch.cat(out)


def run_decode(m, ids, slot=0, tab=None, start=0, graph=True):
    tab = tab or table(len(ids))
    out = []
    for p in range(start, len(ids)):
        m.set_rows(1, [ids[p]], [p], [slot], [tab])
        out.append(m.decode(1, graph=graph)[1][0].clone())
    return torch.stack(out)


@torch.no_grad()
def plain_logits(cfg, W, ids):
    return P.forward(cfg, W, ids, torch.float32)


def model_tol(cfg, W, dtype, ids):
    """Tolerance of whole-model logits of one sequence: fixed in 32-bit; in 16-bit twice what rounding the weights once
    more (to within half a bf16 ulp, at random) does to the plain model - random stacks amplify any rounding, some
    sequences (a head whose maps nearly cancel) more than others."""
    if dtype == F32:
        return 1e-4
    base, errs = plain_logits(cfg, W, ids), []
    for seed in (1, 2, 3):
        g = torch.Generator().manual_seed(seed)
        near = {k: v.float() * (1 + 2.0 ** -8 * (2 * torch.rand(v.shape, generator=g) - 1)) for k, v in W.items()}
        errs.append(rel(plain_logits(cfg, near, ids), base))
    return 2 * max(errs)


# ------------------------------------------------------------------ single mechanisms
@pytest.mark.parametrize("S,W", [(1, 64), (2, 72), (3, 50), (4, 33), (8, 128)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_streams_step(S, W, dtype):
    from coffin_b200.ops import mixers as X
    g = torch.Generator().manual_seed(S * 100 + W)
    r = lambda *s: torch.randn(*s, generator=g).cuda()
    T = 5
    x, y = r(T, S, W), r(T, W).to(dtype)
    read, mix, write, gain = r(S), r(S, S), r(S), r(W)
    new = torch.einsum("st,nsw->ntw", mix.double(), x.double()) + write.double()[None, :, None] * y.double()[:, None]
    norm = lambda u: u / torch.sqrt((u * u).mean(-1, keepdim=True) + 1e-3) * gain.double()
    want = norm(torch.einsum("s,nsw->nw", read.double(), new))
    h = torch.zeros(T, W, dtype=dtype, device="cuda")
    keep = x.clone()
    X.streams_step(x, h, gain=gain, read=read, y=y, mix=mix, write=write, eps=1e-3, store=False)
    assert torch.equal(x, keep) and rel(h, want) < (1e-6 if dtype == F32 else 4e-3)
    X.streams_step(x, h, gain=gain, read=read, y=y, mix=mix, write=write, eps=1e-3)
    assert rel(x, new) < 1e-6 and rel(h, want) < (1e-6 if dtype == F32 else 4e-3)
    rows = torch.tensor([3, 0], dtype=torch.int32, device="cuda")
    h2 = torch.zeros(2, W, dtype=dtype, device="cuda")
    X.streams_step(x, h2, gain=gain, rows=rows, eps=1e-3, store=False)          # plain sum of picked rows
    assert rel(h2, norm(new.sum(1))[[3, 0]]) < (1e-6 if dtype == F32 else 4e-3)


MIX = {
    "delta": Z.delta(), "delta_equal_heads": Z.delta(3, 3, 32, 32, 2), "delta_one_tap": Z.delta(2, 1, 8, 16, 1),
    "delta_wide": Z.delta(2, 1, 72, 64, 5), "delta_odd": Z.delta(2, 2, 10, 7, 3), "delta_128": Z.delta(2, 1, 128, 128, 4),
    "delta_256": Z.delta(1, 1, 256, 40, 4),
    "mlstm": Z.mlstm(), "mlstm_wide": Z.mlstm(2, 64, 136, 14.0), "mlstm_odd": Z.mlstm(5, 9, 13, 3.0), "mlstm_one": Z.mlstm(1, 128, 256, 20.0),
    "attn": Z.attention(), "attn_nocap": Z.attention(softcap=None, every=0), "attn_mqa": Z.attention(5, 1, 24, 16, every=7),
    "attn_equal": Z.attention(2, 2, 64, 128), "attn_wide": Z.attention(2, 1, 128, 256, scale=0.09), "attn_odd": Z.attention(3, 1, 6, 10),
    "attn_many": Z.attention(12, 1, 8, 8, scale=0.5),
}


def mixer_pair(layer, dtype, T, cuts=None, seed=3, h=None, W=None, spike=None):
    """(device, plain) outputs of one mixer on the same rows, cut into portions."""
    cfg = Z.config([layer], width=64, ff=None)
    W = W or Z.weights(cfg, seed)
    m = build(cfg, W, dtype)
    g = torch.Generator().manual_seed(seed + 1)
    h = torch.randn(T, 64, generator=g).to(torch.bfloat16) if h is None else h
    mix = m.layers[0].mixer
    m.zero_state(1)
    outs, at, k = [], 0, 0
    cuts = cuts or [T]
    tab = table(T, first=2, step=2)
    while at < T:
        n = min(cuts[k % len(cuts)], T - at)
        k += 1
        b, _, _ = m.make_batch([([0] * n, at, 1, tab)])
        hb = m.buf("h", n, 64)
        hb.copy_(h[at:at + n])
        act = mix.run(m, b, hb)
        outs.append(m.linear(mix.w_out, act, m.buf("y", n, 64)).float().clone())
        at += n
    ref = P.MIXERS[layer["type"]](h.double(), {k_[7:]: v.double() for k_, v in W.items() if k_.startswith("l0.mix.")}, layer["mixer"],
                                  cfg["norm"]["eps"])
    return torch.cat(outs), ref


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(MIX))
def test_mixer_alone(name, dtype):
    got, ref = mixer_pair(MIX[name], dtype, 83)
    assert rel(got, ref) < TOL[dtype], rel(got, ref)
    assert rel(got[:3], ref[:3]) < 2 * TOL[dtype]                # the first tokens: empty state, empty convolution, m = 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["delta", "mlstm", "attn"])
@pytest.mark.parametrize("cuts", [[1], [2], [3, 1, 17], [16], [15, 33], [64, 65]])
def test_mixer_in_portions(name, dtype, cuts):
    got, ref = mixer_pair(MIX[name], dtype, 150, cuts)
    assert rel(got, ref) < TOL[dtype], rel(got, ref)
    worst = max(rel(got[i:i + 1], ref[i:i + 1]) for i in range(150))
    assert worst < 8 * TOL[dtype], worst


@pytest.mark.parametrize("sizes", [(64, 64), (128, 256), (64, 128), (256, 64), (256, 256), (32, 64), (40, 96)])
@pytest.mark.parametrize("cap", [None, 18.0, 60.0])
def test_prompt_attention_kernels_agree(sizes, cap):
    """tcgen05 (sizes of 64 / 128 / 256), mma.sync and the plain equations on prompts and long portions; peaky scores,
    so that the uncapped form raises its reference maximum again and again."""
    from coffin_b200.ops import kernels as K
    d, e = sizes
    layer = Z.attention(3, 1, d, e, scale=4.0 * d ** -0.5, softcap=cap, every=100)
    for cuts in ([333], [130, 203]):
        got, ref = mixer_pair(layer, BF16, 333, cuts, seed=d + e)
        assert rel(got, ref) < TOL[BF16], (cuts, rel(got, ref))
    K.check_status()
    was, K.ATTN_TC = K.ATTN_TC, False
    try:
        other, _ = mixer_pair(layer, BF16, 333, [130, 203], seed=d + e)
    finally:
        K.ATTN_TC = was
    assert rel(got, other) < 3e-3 and max(rel(got[i:i + 1], other[i:i + 1]) for i in range(0, 333, 7)) < 3e-2


@pytest.mark.parametrize("bias", [-12.0, 12.0])
def test_mlstm_running_maximum_starts_at_zero(bias):
    """With input gates far below (above) zero the denominator's exp(-m) decides the first tokens."""
    layer = Z.mlstm(2, 16, 24, 13.0)
    cfg = Z.config([layer], width=64, ff=None)
    W = Z.weights(cfg, 5)
    W["l0.mix.i.b"] = torch.full_like(W["l0.mix.i.b"], bias)
    for dtype in (F32, BF16):
        got, ref = mixer_pair(layer, dtype, 40, W=W, cuts=[11])
        assert rel(got, ref) < TOL[dtype] * (30 if dtype == F32 and bias < 0 else 2), rel(got, ref)


def test_delta_strong_decays_stay_finite():
    layer = Z.delta(2, 1, 64, 32, 4)
    cfg = Z.config([layer], width=64, ff=None)
    W = Z.weights(cfg, 6)
    W["l0.mix.A_log"] = torch.full_like(W["l0.mix.A_log"], 3.0)           # decays down to exp(-20 * softplus) per token
    W["l0.mix.dt_bias"] = torch.linspace(-6, 4, 128).to(torch.bfloat16)
    for dtype in (F32, BF16):
        got, ref = mixer_pair(layer, dtype, 70, W=W)
        assert torch.isfinite(got).all() and rel(got, ref) < TOL[dtype], rel(got, ref)


# ------------------------------------------------------------------ far keys, page borders
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("mode", ["prompt", "decode", "portions"])
def test_one_far_key_decides_the_attention(dtype, mode):
    """Key ``j`` is made to stand out for every later query (its row and the queries share a direction that the other
    keys lack), at page borders and far back: dropping it, or reading its neighbour, changes the output."""
    layer = Z.attention(4, 2, 16, 24, scale=0.5, softcap=30.0, every=0)
    cfg = Z.config([layer], width=64, ff=None)
    W = Z.weights(cfg, 8)
    for n in ("q", "k"):                       # last input column: only the marked row has it (keys), all rows have a bit (queries)
        w = W[f"l0.mix.{n}"].float() * (0.3 if n == "k" else 0.1)
        w[:, 63] = 0.0
        w[::16, 63] = 6.0 if n == "k" else 0.0
        w[::16, 62] = 2.0 if n == "q" else 0.0
        W[f"l0.mix.{n}"] = w.to(torch.bfloat16)
    T = 200
    cuts = {"prompt": [T], "decode": [1], "portions": [37, 2, 64]}[mode]
    for j in (0, 1, 62, 63, 64, 65, 127, 128, 191):
        g = torch.Generator().manual_seed(j)
        h = torch.randn(T, 64, generator=g)
        h[:, 62], h[:, 63] = 2.0, 0.0
        h[j, 63] = 2.0
        h = h.to(torch.bfloat16)
        got, ref = mixer_pair(layer, dtype, T, cuts, h=h, W=W)
        assert rel(got, ref) < TOL[dtype], (j, rel(got, ref))
        blind = h.clone()
        blind[j, 63] = 0.0                     # the oracle without the mark: what a lost key would look like
        _, lost = mixer_plain(layer, blind, W, cfg)
        assert rel(lost[j + 1:], ref[j + 1:]) > 10 * TOL[dtype], j


def mixer_plain(layer, h, W, cfg):
    return None, P.MIXERS[layer["type"]](h.double(), {k[7:]: v.double() for k, v in W.items() if k.startswith("l0.mix.")},
                                         layer["mixer"], cfg["norm"]["eps"])


def test_query_temperature_steps_where_it_should():
    """The factor changes at position every - 1; a shift by one token shows (large coefficient, peaky scores)."""
    layer = Z.attention(4, 2, 16, 24, scale=0.8, softcap=30.0, coef=3.0, every=50)
    got, ref = mixer_pair(layer, F32, 120, [7, 1, 30])
    for p in (0, 47, 48, 49, 50, 51, 98, 99, 100):
        assert rel(got[p:p + 1], ref[p:p + 1]) < 1e-4, p


# ------------------------------------------------------------------ whole models
CONFIGS = {
    "all": (Z.ALL, 8),
    "one_stream": (Z.config([Z.mlstm(), Z.delta(2, 2, 16, 16, 2)], streams=1, width=40, vocab=51), 5),
    "no_ff": (Z.config([Z.attention(4, 4, 8, 16), Z.mlstm(1, 32, 8), Z.delta()], streams=3, no_mlp=(0, 2), width=65, ff=31, vocab=90), 3),
    "sizes_differ": (Z.config([Z.delta(2, 1, 64, 32), Z.delta(6, 2, 16, 8, 3), Z.attention(2, 1, 64, 64), Z.attention(6, 2, 8, 24, every=5),
                               Z.mlstm(2, 64, 32)], streams=4, width=128, ff=200, vocab=128), 16),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_portions_and_decode_match_the_plain_model(name, dtype):
    cfg, rank = CONFIGS[name]
    W = Z.weights(cfg, 11, rank)
    ids = toks(140, cfg["vocab"], 1)
    ref = plain_logits(cfg, W, ids)
    m = build(cfg, W, dtype)
    tol = model_tol(cfg, W, dtype, ids)
    whole = run_portions(m, ids, [140], slot=2, tab=[4, 9, 6])
    assert rel(whole, ref) < tol, rel(whole, ref)
    for cuts in ([2], [5, 1, 2, 40], [63, 2, 64]):
        got = run_portions(m, ids, cuts, slot=1, tab=[7, 3, 5])
        assert rel(got, ref) < tol, (cuts, rel(got, ref))
    m.zero_state(3)
    dec = run_decode(m, ids[:70], slot=3, tab=[1, 2])
    assert rel(dec, ref[:70]) < tol, rel(dec, ref[:70])
    # prompt, then single tokens through the graph
    m.zero_state(0)
    m.forward_batch([(ids[:61], 0, 0, [11, 12, 13])], [[]])
    dec = run_decode(m, ids, slot=0, tab=[11, 12, 13], start=61)
    assert rel(dec, ref[61:]) < tol, rel(dec, ref[61:])


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_match_each_sequence_alone(dtype):
    cfg, W = Z.ALL, Z.weights(Z.ALL, 12)
    m = build(cfg, W, dtype)
    seqs = [toks(n, cfg["vocab"], n) for n in (90, 33, 5, 130)]
    tabs = [[1, 5], [2], [3], [8, 4, 6]]
    alone = [run_portions(m, s, [len(s)], slot=0, tab=t) for s, t in zip(seqs, tabs)]
    for i in range(4):
        m.zero_state(i)
    at, got, r = [0] * 4, [[] for _ in range(4)], random.Random(5)
    while any(a < len(s) for a, s in zip(at, seqs)):
        live = [i for i in range(4) if at[i] < len(seqs[i]) and r.random() < 0.8]
        r.shuffle(live)
        if not live:
            continue
        items, want = [], []
        for i in live:
            n = min(r.choice((1, 1, 2, 3, 17, 40)), len(seqs[i]) - at[i])
            items.append((seqs[i][at[i]:at[i] + n], at[i], i, tabs[i]))
            want.append(list(range(n)))
        out = m.forward_batch(items, want)
        k = 0
        for i, w in zip(live, want):
            got[i].append(out[k:k + len(w)].clone())
            k += len(w)
            at[i] += len(w)
    for g, a, ids in zip(got, alone, seqs):
        assert rel(torch.cat(g), a) < model_tol(cfg, W, dtype, ids)


@pytest.mark.parametrize("rows", [3, 8, 11, 20])
def test_decode_buckets_match_the_plain_model(rows):
    """Batches of single tokens of unequal sequences, padded to a bucket; above 8 rows on the GEMM path."""
    cfg, W = Z.ALL, Z.weights(Z.ALL, 13)
    m = build(cfg, W, BF16, slots=rows, blocks=3 * rows + 1)
    lens = [3 + 5 * i for i in range(rows)]
    seqs = [toks(n + 6, cfg["vocab"], 50 + n) for n in lens]
    tabs = [[1 + 3 * i, 2 + 3 * i, 3 + 3 * i] for i in range(rows)]
    for i in range(rows):
        m.zero_state(i)
        m.forward_batch([(seqs[i][:lens[i]], 0, i, tabs[i])], [[]])
    M, got = m.bucket_for(rows), []
    for k in range(6):
        m.set_rows(M, [seqs[i][lens[i] + k] for i in range(rows)], [lens[i] + k for i in range(rows)], list(range(rows)), tabs)
        got.append(m.decode(M)[1][:rows].clone())
    for i in range(0, rows, 3):
        ref = plain_logits(cfg, W, seqs[i])[lens[i]:]
        assert rel(torch.stack([g[i] for g in got]), ref) < model_tol(cfg, W, BF16, seqs[i]), i


def test_long_decode_in_32_bit():
    cfg, W = Z.ALL, Z.weights(Z.ALL, 14)
    m = build(cfg, W, F32)
    ids = toks(330, cfg["vocab"], 9)
    m.zero_state(0)
    m.forward_batch([(ids[:10], 0, 0, table(330))], [[]])
    got = run_decode(m, ids, start=10)
    assert rel(got[-40:], plain_logits(cfg, W, ids)[-40:]) < 2e-4


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_trace_replay_reuses_pages_and_slots(dtype):
    """Requests come and go through a pool just large enough; every wanted position equals the plain model."""
    from coffin_b200.engine.replay import TraceReplayer, pool_blocks
    cfg, W = Z.ALL, Z.weights(Z.ALL, 15)
    m = build(cfg, W, dtype, slots=4, blocks=pool_blocks(384), max_seq=384)
    rep = TraceReplayer(m)
    r = random.Random(3)
    seqs = {f"q{i}": toks(n, cfg["vocab"], 70 + i) for i, n in enumerate((100, 60, 64, 20, 65, 128, 2, 90))}
    todo, at, live, used = list(seqs), {}, [], set()
    got = {k: [] for k in seqs}
    steps = 0
    while todo or live:
        held = sum((len(seqs[k]) + 63) // 64 for k in live)
        while todo and len(live) < 4 and held + (len(seqs[todo[0]]) + 63) // 64 <= 6:
            k = todo.pop(0)
            live.append(k)
            at[k] = 0
            held += (len(seqs[k]) + 63) // 64
        entries, end = [], []
        for k in list(live):
            if r.random() < 0.25:
                continue
            n = min(r.choice((1, 2, 5, 31, 64)), len(seqs[k]) - at[k])
            entries.append({"id": k, "tokens": seqs[k][at[k]:at[k] + n], "want": list(range(n))})
            at[k] += n
            if at[k] == len(seqs[k]):
                end.append(k)
        out = rep.step(entries, end)
        used |= {tuple(s.blocks.table) for s in rep.live.values() if s.blocks}
        i = 0
        for e in entries:
            got[e["id"]].append(out[i:i + len(e["want"])])
            i += len(e["want"])
        live = [k for k in live if k not in end]
        steps += 1
    for k, parts in got.items():
        assert rel(torch.cat(parts), plain_logits(cfg, W, seqs[k])) < model_tol(cfg, W, dtype, seqs[k]), k
    assert not rep.live and rep.engine.bm.pool.used_blocks == 0 and len(rep.engine.scheduler.free_slots) == 4


# ------------------------------------------------------------------ the engine's own path
def plain_greedy(cfg, W, prompt, n):
    ids, out = list(prompt), []
    for _ in range(n):
        out.append(int(plain_logits(cfg, W, ids)[-1].argmax()))
        ids.append(out[-1])
    return out


@pytest.mark.parametrize("mixed", [True, False])
def test_greedy_generation_through_the_engine(mixed):
    from coffin_b200.engine.config import EngineConfig
    from coffin_b200.engine.llm_engine import LLMEngine
    from coffin_b200.engine.sequence import SamplingParams
    cfg, W = Z.ALL, Z.weights(Z.ALL, 16)
    m = build(cfg, W, F32, slots=3, blocks=24, max_seq=256)
    eng = LLMEngine(m, EngineConfig(max_seq=256, max_num_seqs=3, chunk=48, prefill_quantum=48, max_num_batched_tokens=64,
                                    mixed_batch=mixed, snapshot_interval=64))
    prompts = [toks(n, cfg["vocab"], 90 + n) for n in (70, 9, 40, 130, 3)]
    params = SamplingParams(max_tokens=10, ignore_eos=True)
    seqs = eng.generate(prompts, params)
    prompts.append(prompts[3][:128] + [7])                     # shares a cached prefix: pages by reference, states restored
    seqs += eng.generate(prompts[-1:], params)
    assert (eng.runner.n_mixed_steps > 0) == mixed and eng.runner.n_cached_tokens > 0
    for s, p in zip(seqs, prompts):
        assert s.output == plain_greedy(cfg, W, p, 10)


def test_llm_entry_point_generates_the_engines_tokens(tmp_path):
    from coffin_b200.config import load_config
    from coffin_b200.engine.llm import LLM
    from coffin_b200.models.zufilorn.config import ZufilornConfig
    from coffin_b200.weights.init import save_checkpoint
    cfg, W = Z.ALL, Z.weights(Z.ALL, 17)
    save_checkpoint(ZufilornConfig.from_hf(cfg), W, tmp_path)
    assert load_config(tmp_path).layer_types == ("channel_delta", "mlstm", "attention")
    llm = LLM.from_pretrained(tmp_path, max_seq=256, dtype=torch.float32)
    p = toks(50, cfg["vocab"], 4)
    out = llm.generate(p, max_new_tokens=12)
    assert out.tokens == plain_greedy(cfg, W, p, 12)
    first = llm.device_prefill(torch.tensor(p).cuda())
    assert [int(first[0])] + llm.device_decode(first, 11).tolist() == out.tokens


def test_bad_batches_stop_on_the_host():
    m = build(Z.ALL, Z.weights(Z.ALL, 18), BF16, slots=2, blocks=4)
    for item in (([1, 2], 63, 0, [1]), ([1], 0, 2, [1]), ([1], 0, 0, [9]), ([1], 640, 0, list(range(10)))):
        with pytest.raises(ValueError):
            m.forward_batch([item], [[]])
    with pytest.raises(ValueError):
        m.forward_batch([([1], 0, 0, [1]), ([2], 0, 0, [2])], [[], []])


def test_serving_process_answers_with_the_plain_models_tokens(tmp_path):
    """The resident engine process built from a checkpoint directory by the command line's own builder: greedy and
    sampled requests, several at once."""
    import threading
    from coffin_b200.entrypoints.cli.runtime import build_server, parser
    from coffin_b200.models.zufilorn.config import ZufilornConfig
    from coffin_b200.serving.transport import call, serve
    from coffin_b200.weights.init import save_checkpoint
    cfg = Z.config([Z.mlstm(), Z.delta(), Z.attention()], vocab=300)
    W = Z.weights(cfg, 19)
    save_checkpoint(ZufilornConfig.from_hf(cfg), W, tmp_path / "model")
    srv = build_server(parser().parse_args(["--serve", "--model", str(tmp_path / "model"), "--max-seq", "256", "--max-num-seqs", "4"]))
    sock, ready = str(tmp_path / "s.sock"), threading.Event()
    t = threading.Thread(target=serve, args=(srv, sock), kwargs={"ready": ready}, daemon=True)
    t.start()
    assert ready.wait(60)
    try:
        prompts = [toks(n, 256, n) for n in (20, 75, 3)]
        reps = [None] * 3

        def ask(i):
            reps[i] = call(sock, {"op": "generate", "tokens": prompts[i], "max_new": 6, "ignore_eos": True})
        threads = [threading.Thread(target=ask, args=(i,)) for i in range(3)]
        for th in threads:
            th.start()
        for th in threads:
            th.join(60)
        for p, rep in zip(prompts, reps):
            assert rep["ok"] and rep["n_new"] == 6
            ids = list(p)
            for tok in rep["tokens"]:                  # 16-bit: the token has to be among the plain model's near-best
                lg = plain_logits(cfg, W, ids)[-1]
                assert lg.max() - lg[tok] < 0.15 * lg.std(), rep["tokens"]
                ids.append(tok)
        warm = call(sock, {"op": "generate", "tokens": prompts[0], "max_new": 6, "temperature": 0.8, "seed": 3, "ignore_eos": True})
        assert warm["ok"] and all(0 <= x < 300 for x in warm["tokens"])
    finally:
        call(sock, {"op": "stop"})
        t.join(timeout=20)

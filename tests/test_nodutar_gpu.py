"""Nodutar on the device against the plain restatement of its equations (``plain_nodutar.py``)."""
import random

import pytest
import torch

import nodutar_cases as S
import plain_nodutar as P
from test_fasolorn_gpu import check, randn, row_error, slots_of
from test_zufilorn_gpu import rel, run_decode, run_portions, table, toks

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
# rms of the error over the rms of the value: 32-bit mode, serving mode
TOL = {F32: 2e-5, BF16: 2e-2}
EPS = 3e-5


def build(cfg, W, dtype=F32, slots=4, blocks=40, max_seq=640, **kw):
    from coffin_b200.models import build_model
    from coffin_b200.models.nodutar.config import NodutarConfig
    return build_model(NodutarConfig.from_hf(cfg), W, device="cuda", dtype=dtype, num_slots=slots, num_blocks=blocks, max_seq=max_seq, **kw)


@torch.no_grad()
def plain_logits(cfg, W, ids):
    return P.forward(cfg, W, ids, torch.float32)


def model_tol(cfg, W, dtype, ids):
    """Tolerance of whole-model logits of one sequence: fixed in 32-bit; in 16-bit twice what rounding the weights once
    more (to within half a bf16 ulp, at random) does to the plain model."""
    if dtype == F32:
        return 1e-4
    base, errs = plain_logits(cfg, W, ids), []
    for seed in (1, 2):
        g = torch.Generator().manual_seed(seed)
        near = {k: v.float() * (1 + 2.0 ** -8 * (2 * torch.rand(v.shape, generator=g) - 1)) for k, v in W.items()}
        errs.append(row_error(plain_logits(cfg, near, ids), base))
    return 2 * max(errs)


# ------------------------------------------------------------------ the residual
@pytest.mark.parametrize("T,W", [(1, 64), (1, 2048), (5, 72), (3, 50), (200, 512), (2, 33), (1, 1030), (2, 6000), (1, 9001)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_residual_step_norms_what_it_adds_and_repeats_the_embedding(T, W, dtype):
    from coffin_b200.ops import mixers as X
    W8, k = (W + 7) // 8 * 8, 4
    x, gain, post = randn(1, T, W).cuda() * 3, randn(3, W).cuda(), randn(4, W).cuda()
    y, h = (torch.zeros(T, W8, dtype=dtype, device="cuda") for _ in range(2))
    y[:, :W] = (randn(2, T, W) * 7).to(dtype)
    E, tok = randn(5, 11, W).to(dtype).cuda(), torch.randint(0, 11, (T,), generator=torch.Generator().manual_seed(6)).cuda()
    tol = 2e-6 if dtype == F32 else 4e-3
    d = lambda t: t.double().cpu()
    norm = lambda u, g: P.unit_rms(d(u), 1e-3) * d(g)
    keep = x.clone()
    want = d(x) + norm(y[:, :W], post)
    X.residual_step(x, h, gain=gain, y=y, post=post, eps=1e-3, store=False)
    assert torch.equal(x, keep) and rel(h[:, :W], norm(want, gain)) < tol
    rows = torch.arange(T - 1, -1, -1, dtype=torch.int32, device="cuda")[:2]
    h2 = torch.zeros(rows.numel(), W8, dtype=dtype, device="cuda")
    X.residual_step(x, h2, gain=gain, y=y, post=post, rows=rows, store=False, eps=1e-3)
    assert rel(h2[:, :W], norm(want, gain)[rows.long().cpu()]) < tol
    X.residual_step(x, h, gain=gain, y=y, post=post, again=(E, tok), eps=1e-3)
    want += d(E[tok])
    assert rel(x, want) < 1e-6 and rel(h[:, :W], norm(want, gain)) < tol
    X.residual_step(x, h, gain=gain, again=(E, tok), eps=1e-3)                              # the embedding alone
    want += d(E[tok])
    assert rel(x, want) < 1e-6 and rel(h[:, :W], norm(want, gain)) < tol
    ys = torch.zeros(T * k, W8, dtype=dtype, device="cuda")
    ys[:, :W] = randn(7, T * k, W).to(dtype)
    pos = torch.randperm(T * k, generator=torch.Generator().manual_seed(1)).view(T, k).int()
    pos[:, 1] = -1
    w = randn(8, T, k).abs()
    merged = sum(d(w[:, j, None]) * d(ys[pos[:, j].long().clamp(min=0).cuda(), :W]) for j in (0, 2, 3))
    X.residual_step(x, None, experts=(ys, pos.cuda(), w.cuda(), None, None), post=post, eps=1e-3)
    assert rel(x, want + norm(merged, post)) < 1e-6
    assert (h[:, W:] == 0).all()


# ------------------------------------------------------------------ routing and experts
@pytest.mark.parametrize("E,top", [(7, 3), (4, 1), (5, 5), (128, 8), (512, 32), (1, 1)])
@pytest.mark.parametrize("T", [1, 8, 33, 100])
def test_routing_by_logits(E, top, T):
    from coffin_b200.ops import routed as R
    r = R.Router(E, 0, top, 1.0, 0, True)
    z, b = randn(1, T, E) * 2, randn(2, E)
    zd = torch.zeros(T, E + 3, device="cuda")
    zd[:, :E] = z
    ref_i, ref_w = P.route(z.double() + b.double(), top)
    idx, w, idw = slots_of(r, T)
    for units in (False, True)[:1 + (T <= R.UNIT_ROWS)]:
        if units:
            R.route_units(r, zd, b.cuda(), None, idx, w, idw, torch.zeros(R.meta_size(r, T), dtype=torch.int32, device="cuda"))
        else:
            R.route(r, zd, b.cuda(), None, idx, w, idw)
        for t in range(T):
            want = dict(zip(ref_i[t].tolist(), ref_w[t].tolist()))
            got = dict(zip(idx[t].tolist(), w[t].tolist()))
            assert set(got) == set(want) and all(abs(got[i] - want[i]) < 1e-5 for i in got)


def test_bias_takes_part_in_choice_and_weights():
    from coffin_b200.ops import routed as R
    r = R.Router(4, 0, 2, 1.0, 0, True)
    z = torch.tensor([[3.0, 2.0, 0.0, -1.0], [200.0, -200.0, -150.0, -300.0]]).cuda()       # weights far apart underflow, the choice does not
    for b, chosen in (([0.0] * 4, ((0, 1), (0, 2))), ([0.0, 0.0, 0.0, 5.0], ((3, 0), (0, 2))), ([-9.0, 0.0, 0.0, 0.0], ((1, 2), (0, 2)))):
        idx, w, idw = slots_of(r, 2)
        R.route(r, z, torch.tensor(b).cuda(), None, idx, w, idw)
        s = z.cpu().double() + torch.tensor(b).double()
        for t in range(2):
            assert idx[t].tolist() == list(chosen[t])
            assert torch.allclose(w[t].cpu().double(), torch.softmax(s[t, list(chosen[t])], 0), atol=1e-6)


@pytest.mark.parametrize("N,Kd", [(56, 72), (512, 2048), (13, 8), (40, 1032)])
@pytest.mark.parametrize("T,top", [(1, 3), (8, 3), (40, 2), (64, 1)])
def test_gated_unit_products(N, Kd, T, top):
    from coffin_b200.ops import kernels as K
    from coffin_b200.ops import routed as R
    r = R.Router(9, 0, top, 1.0, 0, True)
    W, x = (randn(1, 9, 2 * N, Kd) * Kd ** -0.5).bfloat16(), randn(2, T, Kd).bfloat16()
    idx, w, idw = slots_of(r, T)
    meta = torch.zeros(R.meta_size(r, T), dtype=torch.int32, device="cuda")
    d = R.route_units(r, (randn(3, T, 9) * 3).cuda(), torch.zeros(9).cuda(), None, idx, w, idw, meta)
    e, pos = idx.cpu().view(-1).long(), d["pos"].cpu().long()
    src = torch.arange(T).repeat_interleave(top)
    gu = torch.einsum("snk,sk->sn", W.double()[e], x.double()[src])
    ref = P.silu(gu[:, :N]) * gu[:, N:]
    for dtype, tol in ((F32, 2e-6), (BF16, 4e-3)):
        out = torch.full((T * top, N), 3.0, dtype=dtype, device="cuda")
        Wd, xd = W.to(dtype).cuda(), x.to(dtype).cuda()
        R.unit_linear(Wd, xd, out, d, rows=T, gather=True, swiglu=True)
        assert rel(out[pos], ref) < tol
        rows = torch.zeros(T * top, Kd, dtype=dtype, device="cuda")
        rows[pos] = xd[src]
        R.unit_linear(Wd, rows, out, d, rows=T, gather=False, swiglu=True)
        assert rel(out[pos], ref) < tol
    K.check_status()


MOE = {"some": S.moe(), "one_of_many": S.moe(30, 1, 16), "all_of_them": S.moe(3, 3, 32), "large": S.moe(6, 2, 264), "odd": S.moe(5, 2, 13), "one": S.moe(1, 1, 24)}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(MOE))
@pytest.mark.parametrize("width", [72, 65])
def test_routed_feed_forward(name, dtype, width):
    """Few rows, units, grouped GEMM: every count of rows gives the plain result."""
    from coffin_b200.ops import mixers as X
    cfg = S.config([S.attention()], [MOE[name]], width=width)
    W = S.weights(cfg, 5)
    m = build(cfg, W, dtype)
    ff = {k[7:]: v.double() for k, v in W.items() if k.startswith("l0.mlp.")}
    h = randn(6, 300, width).bfloat16()
    ref = P.experts(h.double(), ff, MOE[name])
    for T in (1, 3, 8, 9, 33, 64, 65, 300):
        b, _, _ = m.make_batch([([0] * T, 0, 0, table(T))])
        hb = m.buf("h", T, (width + 7) // 8 * 8)
        hb[:, :width].copy_(h[300 - T:])
        x = torch.zeros(T, width, device="cuda")
        X.residual_step(x, None, **m.layers[0].routed.run(m, b, hb))
        assert (rel if dtype == F32 else row_error)(x, ref[300 - T:]) < TOL[dtype], T
    m.check_status()


# ------------------------------------------------------------------ mixers alone
def left_only(*a, **kw):
    return S.parallel(*a, **dict({"rs": 0.0}, **kw))


def right_only(*mem, chunk=20):
    return S.parallel(2, 1, 8, 8, chunk, 4, mem=mem, ls=0.0, rs=1.3)


MIX = {
    "parallel": S.parallel(), "parallel_negative_scale": S.parallel(ls=-0.5, rs=0.25),
    "left": left_only(), "left_one_head": left_only(1, 1, 8, 8, 3, 4), "no_chunks": left_only(chunk=0), "chunk_1": left_only(chunk=1), "chunk_64": left_only(chunk=64),
    "chunk_65": left_only(chunk=65), "chunk_63": left_only(4, 4, 16, 16, 63), "chunk_far": left_only(chunk=500), "no_rotation": left_only(rot=0),
    "all_rotated": left_only(4, 2, 24, 16, 40, 24), "groups_of_12": left_only(24, 2, 16, 24, 50, 8), "equal_turns": left_only(3, 3, 16, 16, 70, 16),
    "64_128": left_only(4, 2, 64, 128, 50, 64), "128": left_only(4, 1, 128, 128, 90, 64, scale=0.1), "192_64": left_only(2, 2, 192, 64, 40, 10, scale=0.07),
    "256": left_only(2, 1, 256, 256, 70, 64, scale=0.06), "odd": left_only(3, 3, 7, 10, 20, 6), "odd_values": left_only(4, 2, 16, 14, 33, 16),
    "large_values": left_only(2, 1, 32, 300, 40, 8), "192_192": left_only(2, 1, 192, 192, 70, 64, scale=0.07),
    "right": right_only(3, 40, 24), "right_one": right_only(1, 8, 8), "right_128": right_only(2, 128, 128), "right_256": right_only(1, 256, 64), "right_odd": right_only(3, 10, 7),
    "right_wide": right_only(2, 24, 136), "right_tall": right_only(2, 200, 8), "right_64_48": right_only(5, 64, 48),
    "attention": S.attention(), "attention_one": S.attention(1, 1, 8), "attention_equal": S.attention(3, 3, 16), "attention_many": S.attention(24, 2, 24), "attention_64": S.attention(4, 2, 64, 0.2),
    "attention_128": S.attention(4, 1, 128, 0.2), "attention_192": S.attention(2, 1, 192, 0.1), "attention_256": S.attention(2, 2, 256, 0.1), "attention_96": S.attention(4, 2, 96, 0.15),
    "attention_odd": S.attention(3, 1, 13), "attention_large": S.attention(2, 1, 300, 0.1), "attention_32": S.attention(20, 4, 32), "attention_minus": S.attention(4, 2, 64, -0.2),
}


def plain_mixer(layer, W, h, **other):
    """``other``: changed constants of the left half (a mistake planted in the equations)."""
    mix, m = {k[7:]: v.double() for k, v in W.items() if k.startswith("l0.mix.")}, layer["mixer"]
    if layer["type"] == "parallel":
        return P.parallel(h.double(), mix, dict(m, left=dict(m["left"], **other)), EPS)
    return P.distance_attention(h.double(), mix, m, EPS)


def mixer_pair(layer, dtype, T, cuts=None, seed=3, h=None, W=None):
    """(device, plain) outputs of one mixer on the same rows, cut into portions."""
    cfg = S.config([layer], [None], width=64, eps=EPS)
    W = W or S.weights(cfg, seed)
    m = build(cfg, W, dtype)
    h = randn(seed + 1, T, 64).bfloat16() if h is None else h
    mix, tab, cuts = m.layers[0].mixer, table(T, first=2, step=2), cuts or [T]
    m.zero_state(1)
    outs, at, k = [], 0, 0
    while at < T:
        n = min(cuts[k % len(cuts)], T - at)
        k += 1
        b, _, _ = m.make_batch([([0] * n, at, 1, tab)])
        hb = m.buf("h", n, 64)
        hb.copy_(h[at:at + n])
        outs.append(m.linear(mix.w_out, mix.run(m, b, hb), m.buf("y", n, 64)).float().clone())
        at += n
    m.check_status()
    return torch.cat(outs), plain_mixer(layer, W, h)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(MIX))
def test_mixer_alone(name, dtype):
    for cuts in (None, [1]):
        got, ref = mixer_pair(MIX[name], dtype, 150, cuts)
        assert rel(got, ref) < TOL[dtype], (cuts, rel(got, ref))
        assert rel(got[:3], ref[:3]) < 2 * TOL[dtype]               # the first tokens: one key, two, three


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["parallel", "128", "odd", "groups_of_12", "chunk_65", "right_128", "right_odd", "attention", "attention_128", "attention_odd", "attention_many"])
@pytest.mark.parametrize("cuts", [[2], [3, 1, 17], [24, 25], [64], [63, 2, 65], [130, 3]])
def test_mixer_in_portions(name, dtype, cuts):
    got, ref = mixer_pair(MIX[name], dtype, 200, cuts)
    assert rel(got, ref) < TOL[dtype], rel(got, ref)
    worst = max(rel(got[i:i + 1], ref[i:i + 1]) for i in range(200))
    assert worst < 8 * TOL[dtype], worst


@pytest.mark.parametrize("layer", [left_only(4, 2, 64, 64, 100, 32, scale=0.6), left_only(2, 1, 128, 256, 129, 128, scale=0.4), left_only(2, 2, 64, 128, 64, 8, scale=0.6),
                                   left_only(4, 1, 256, 64, 300, 64, scale=0.3), left_only(2, 1, 192, 192, 96, 64, scale=0.3), S.attention(4, 2, 64, 0.8), S.attention(2, 1, 128, 0.6),
                                   S.attention(2, 1, 192, 0.4), S.attention(2, 2, 256, 0.3), left_only(4, 2, 64, 64, 100, 32, scale=0.1), left_only(4, 2, 128, 128, 200, 64, scale=0.06),
                                   left_only(2, 1, 256, 128, 0, 64, scale=0.03), left_only(2, 2, 192, 192, 70, 64, scale=0.03), S.attention(4, 2, 64, 0.5), S.attention(2, 1, 128, 0.25),
                                   S.attention(2, 1, 192, 0.15), S.attention(2, 2, 256, 0.12)])
def test_prompt_attention_kernels_agree(layer):
    """tcgen05, mma.sync and the plain equations on prompts and long portions; peaky scores, so that the reference maximum is
    raised again and again, and chunks that leave whole pages of a tile to some of its rows."""
    from coffin_b200.ops import kernels as K
    got = {}
    for tc in (True, False):
        was, K.ATTN_TC = K.ATTN_TC, tc
        try:
            for cuts in ([450], [130, 203]):
                got[tc], ref = mixer_pair(layer, BF16, 450, cuts, seed=9)
                assert rel(got[tc], ref) < 1.5 * TOL[BF16], (tc, cuts, rel(got[tc], ref))
        finally:
            K.ATTN_TC = was
    assert rel(got[True], got[False]) < 4e-3


@pytest.mark.parametrize("nsplit", [1, 2, 3, 7])
@pytest.mark.parametrize("kind", ["left", "attention"])
def test_key_splits(kind, nsplit, monkeypatch):
    """More splits than pages, splits that start in the middle of the walk, chunks that start in the middle of a page."""
    from coffin_b200.ops import mixers as X
    monkeypatch.setattr(X.AttnMaps, "decode_splits", lambda self, rows: nsplit)
    for chunk in (1, 63, 64, 65, 130, 200) if kind == "left" else (0,):
        layer = left_only(4, 2, 16, 24, chunk, 8) if kind == "left" else S.attention(4, 2, 24)
        got, ref = mixer_pair(layer, BF16, 230, [190, 1])
        assert rel(got[190:], ref[190:]) < TOL[BF16], chunk


@pytest.mark.parametrize("layer", [left_only(6, 2, 64, 64, 150, 32, scale=0.1), left_only(3, 1, 32, 256, 0, 8, scale=0.2), left_only(4, 2, 256, 64, 90, 8, scale=0.03), S.attention(4, 2, 24),
                                   S.attention(12, 1, 64, 0.4), S.attention(2, 1, 256, 0.1)])
def test_bounded_scores_need_no_running_maximum(layer, monkeypatch):
    """The same results with the bound as the softmax's reference and with running maxima, on prompts, portions and decode steps of
    one and of several splits; scores at the bound itself and far below it."""
    from coffin_b200.ops import mixers as X
    W = S.weights(S.config([layer], [None], width=64), 3)
    pre = "l0.mix.left." if layer["type"] == "parallel" else "l0.mix."
    for n in ("q", "k"):                                           # one direction dominates: scores near plus and minus the bound
        W[pre + n] = (W[pre + n].float() * 0.3 + 2.0 * torch.randn(W[pre + n].shape[0], 1) * torch.eye(64)[:1]).bfloat16()
    h = randn(4, 230, 64)
    h[:, 0] *= 3
    h = h.bfloat16()
    for cuts in ([230], [140, 1, 2], [1]):
        for ns in (1, 3):
            monkeypatch.setattr(X.AttnMaps, "decode_splits", lambda self, rows: ns)
            a, ref = mixer_pair(layer, BF16, 230, cuts, h=h, W=W)
            with monkeypatch.context() as mp:
                mp.setattr(X.AttnMaps, "_bound", staticmethod(lambda *x: 0.0))
                b, _ = mixer_pair(layer, BF16, 230, cuts, h=h, W=W)
            assert rel(a, ref) < 2 * TOL[BF16] and rel(b, ref) < 2 * TOL[BF16] and rel(a, b) < 6e-3, (cuts, ns, rel(a, ref), rel(a, b))


def standout(kind, chunk=0):
    """A layer and weights with which a key whose row has a mark (column 63) stands out for every query (column 62 of all rows)."""
    layer = left_only(4, 2, 16, 24, chunk, 8, scale=0.8) if kind == "left" else S.attention(4, 2, 16, 0.9)
    pre, W = ("l0.mix.left." if kind == "left" else "l0.mix."), S.weights(S.config([layer], [None], width=64), 8)
    q, k = W[pre + "q"].float() * 0.2, W[pre + "k"].float()
    q[:, 62:], k[:, 62:] = 0.0, 0.0
    for hd in range(4):                                            # column 9 of a head does not turn
        q[hd * 16 + 9] = 0.0
        q[hd * 16 + 9, 62] = 4.0
    for g in range(2):
        k[g * 16 + 9] = 0.0
        k[g * 16 + 9, 63] = 6.0
    W[pre + "q"], W[pre + "k"] = q.bfloat16(), k.bfloat16()
    if kind == "left":
        W[pre + "q.norm"], W[pre + "k.norm"] = torch.ones(16).bfloat16(), torch.ones(16).bfloat16()
    return layer, W


def marked(j, T):
    h = randn(j, T, 64)
    h[:, 62], h[:, 63] = 2.0, 0.0
    h[j, 63] = 2.0
    return h.bfloat16()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("mode", ["prompt", "decode", "portions"])
def test_one_key_decides_until_its_chunk_ends(mode, dtype):
    """Key ``j`` stands out for every query that sees it.  Chunks that end before, at and after page borders; a chunk one token
    longer or shorter, a chunk counted from a portion's start, or a missing key would show in single rows."""
    T, cuts = 200, {"prompt": [200], "decode": [1], "portions": [37, 2, 64, 1]}[mode]
    for size, js in ((40, (0, 1, 39, 40, 63, 64, 150)), (64, (0, 63, 64, 65)), (65, (0, 64, 65, 129)), (130, (0, 61, 129)), (2, (63, 64)), (96, (95, 96, 100))):
        layer, W = standout("left", size)
        for j in js:
            h = marked(j, T)
            got, ref = mixer_pair(layer, dtype, T, cuts, h=h, W=W)
            last = min(T, (j // size + 1) * size) - 1              # the last row that sees it
            for i in (i for i in (j - 1, j, j + 1, last - 1, last, last + 1, last + 2) if 0 <= i < T):
                assert rel(got[i:i + 1], ref[i:i + 1]) < 4 * TOL[dtype], (size, j, i, rel(got[i:i + 1], ref[i:i + 1]))
            assert rel(got, ref) < 2 * TOL[dtype]
            if last + 1 < T and j < size:
                longer, shorter = (plain_mixer(layer, W, h, mask={"size": size + d}) for d in (1, -1))
                assert rel(longer[last + 1], ref[last + 1]) > 20 * TOL[dtype], (size, j)
                assert j == last or rel(shorter[last], ref[last]) > 20 * TOL[dtype], (size, j)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("mode", ["prompt", "decode", "portions"])
def test_one_far_key_decides_the_attention(mode, dtype):
    """A key that stands out hundreds of tokens back, at page borders and among the first tokens; without it rows would
    differ plainly."""
    T, cuts = 330, {"prompt": [330], "decode": [1], "portions": [129, 2, 64, 1]}[mode]
    layer, W = standout("attention")
    for j in (0, 1, 63, 64, 65, 127, 200):
        h = marked(j, T)
        got, ref = mixer_pair(layer, dtype, T, cuts, h=h, W=W)
        for i in (i for i in (j, j + 1, j + 2, 128, 255, 256, T - 1) if i >= j):
            assert rel(got[i:i + 1], ref[i:i + 1]) < 4 * TOL[dtype], (j, i)
        assert rel(got, ref) < 2 * TOL[dtype]
        blind = h.clone()
        blind[j, 63] = 0.0
        assert rel(plain_mixer(layer, W, blind)[T - 1], ref[T - 1]) > 20 * TOL[dtype]


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_penalty_of_the_distance(dtype):
    """Steep, flat and absent penalties, near and far; a distance one off would show."""
    layer = S.attention(4, 2, 32, 0.4)
    W = S.weights(S.config([layer], [None], width=64), 5)
    for r1, r2 in ((3.0, 5.0), (0.5, 0.002), (1.0, 0.0), (0.0, 1.0), (-0.4, 0.3), (8.0, 0.05)):
        W["l0.mix.r1"], W["l0.mix.r2"] = torch.full((4,), r1).bfloat16(), torch.tensor([r2, 2 * r2, r2, r2 / 2]).bfloat16()
        for cuts in ([300], [1], [130, 2, 31]):
            got, ref = mixer_pair(layer, dtype, 300, cuts, W=W)
            assert rel(got, ref) < TOL[dtype], (r1, r2, cuts)
            assert rel(got[290:], ref[290:]) < 2 * TOL[dtype]
    W["l0.mix.r1"], W["l0.mix.r2"] = torch.full((4,), 3.0).bfloat16(), torch.full((4,), 5.0).bfloat16()
    ref, was = plain_mixer(layer, W, randn(4, 60, 64).bfloat16()), P.log_distance
    try:
        P.log_distance = lambda T, r1, r2, dt: r1 * torch.log(1 + r2 * ((torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0) + 1).to(dt))
        assert rel(plain_mixer(layer, W, randn(4, 60, 64).bfloat16()), ref) > 10 * TOL[BF16]
    finally:
        P.log_distance = was


def test_values_are_the_keys_ahead_of_their_norm():
    """Keys of very different lengths: equal in scores, not as values."""
    layer = S.attention(2, 1, 64, 0.3)
    W, h = S.weights(S.config([layer], [None], width=64), 6), randn(9, 200, 64)
    h *= torch.logspace(-1.5, 1.5, 200)[torch.randperm(200, generator=torch.Generator().manual_seed(1))][:, None]
    h = h.bfloat16()
    for dtype in (F32, BF16):
        for cuts in ([200], [1], [130, 2, 5]):
            got, ref = mixer_pair(layer, dtype, 200, cuts, h=h, W=W)
            assert rel(got, ref) < TOL[dtype], (dtype, cuts)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_values_turn_with_their_position_and_heads_turn_back(dtype):
    """Leaving out either turn, or both, would show."""
    layer = left_only(4, 2, 16, 32, 0, 8, base=50.0, scale=0.2)
    W, h = S.weights(S.config([layer], [None], width=64), 6), randn(4, 150, 64).bfloat16()
    for cuts in ([150], [1], [70, 2, 3]):
        got, ref = mixer_pair(layer, dtype, 150, cuts, h=h, W=W)
        assert rel(got, ref) < TOL[dtype]
    was = P.rotate_pairs
    try:
        for skip in ({1}, {-1}, {1, -1}):                          # of the whole values (32 columns), by the direction of the turn
            P.rotate_pairs = lambda x, dims, base, sign=1: x if dims == 32 and sign in skip else was(x, dims, base, sign)
            assert rel(plain_mixer(layer, W, h), ref) > 10 * TOL[BF16], skip
    finally:
        P.rotate_pairs = was


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("mem", [(2, 32, 24), (1, 128, 64), (2, 20, 6)])
def test_forget_gates_from_none_to_all(mem, dtype):
    """States that are overwritten by every token, kept over hundreds of tokens, or held by the lower bound alone."""
    layer = right_only(*mem)
    W, n = S.weights(S.config([layer], [None], width=64), 7), mem[0] * mem[1]
    b, low = "l0.mix.right.f.b", "l0.mix.right.lower"
    mixed = torch.linspace(-30, 12, n)
    for bias, lower in ((torch.full((n,), -25.0), torch.zeros(n)), (torch.full((n,), 9.0), torch.zeros(n)), (torch.full((n,), -40.0), torch.full((n,), 0.97)),
                        (mixed, torch.zeros(n)), (mixed.flip(0), torch.linspace(0, 0.996, n)), (torch.full((n,), -120.0), torch.zeros(n))):
        W[b], W[low] = bias.bfloat16(), lower.bfloat16()
        for cuts in ([230], [1], [100, 2, 17, 16]):
            got, ref = mixer_pair(layer, dtype, 230, cuts, W=W)
            assert torch.isfinite(got).all() and rel(got, ref) < TOL[dtype], (float(bias[0]), cuts, rel(got, ref))


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_a_token_is_remembered_across_portions(dtype):
    """One token writes far more than the others into slow channels; a state lost between portions would show at the end."""
    layer = right_only(2, 32, 24)
    W, T = S.weights(S.config([layer], [None], width=64), 8), 300
    W["l0.mix.right.f.b"], W["l0.mix.right.lower"] = torch.full((64,), 6.0).bfloat16(), torch.zeros(64).bfloat16()
    W["l0.mix.right.f"][:, 63] = -2.0
    for j in (0, 15, 16, 63, 64, 130):
        h = randn(j, T, 64)
        h[:, 63] = 0.0
        h[j, 63] = 4.0
        h = h.bfloat16()
        for cuts in ([300], [1], [64], [16, 1, 2, 15]):
            got, ref = mixer_pair(layer, dtype, T, cuts, h=h, W=W)
            assert rel(got[j:], ref[j:]) < TOL[dtype] and rel(got[-1], ref[-1]) < 3 * TOL[dtype], (j, cuts)
        gone = h.clone()
        gone[j] = 0.0
        assert rel(plain_mixer(layer, W, gone)[-1], ref[-1]) > 10 * TOL[BF16]


@pytest.mark.parametrize("mem", [(2, 32, 24), (1, 128, 64), (3, 200, 40), (1, 16, 72)])
def test_long_portions_of_unequal_length_scan_in_blocks(mem):
    """One forward over portions from two tokens to hundreds, some continuing a state; memories that outlast a block of the scan."""
    layer = right_only(*mem)
    W, n = S.weights(S.config([layer], [None], width=64, eps=EPS), 7), mem[0] * mem[1]
    W["l0.mix.right.f.b"] = torch.linspace(2, 8, n).bfloat16()
    m = build(S.config([layer], [None], width=64, eps=EPS), W, BF16, blocks=60, max_seq=1300)
    hs = [randn(30 + i, t, 64).bfloat16() for i, t in enumerate((900, 2, 300, 129))]
    for i in range(4):
        m.zero_state(i)
    mix, tabs = m.layers[0].mixer, [table(900, 1), table(2, 20), table(300, 22), table(129, 30)]
    at, got = [0] * 4, [[] for _ in range(4)]
    for cuts in ((0, 2, 0, 129), (640, 0, 17, 0), (260, 0, 283, 0)):
        live = [i for i in range(4) if cuts[i]]
        b, _, first = m.make_batch([([0] * cuts[i], at[i], i, tabs[i]) for i in live])
        hb = m.buf("h", b.T, 64)
        for k, i in enumerate(live):
            hb[first[k]:first[k] + cuts[i]].copy_(hs[i][at[i]:at[i] + cuts[i]])
        y = m.linear(mix.w_out, mix.run(m, b, hb), m.buf("y", b.T, 64)).float().clone()
        for k, i in enumerate(live):
            got[i].append(y[first[k]:first[k] + cuts[i]])
            at[i] += cuts[i]
    m.check_status()
    for g, h in zip(got, hs):
        ref, g = plain_mixer(layer, W, h), torch.cat(g)
        assert rel(g, ref) < TOL[BF16] and max(rel(g[i:i + 16], ref[i:i + 16]) for i in range(0, len(h), 16)) < 2 * TOL[BF16]


# ------------------------------------------------------------------ whole models
CONFIGS = {
    "all": S.ALL,
    "narrow": S.config([S.parallel(2, 1, 8, 8, 30, 4, mem=(1, 8, 8)), S.attention(2, 1, 8)], [S.moe(3, 1, 8), S.moe(2, 2, 24)], None, width=40, vocab=51),
    "no_ff": S.config([S.attention(4, 4, 8), S.parallel(4, 2, 8, 8, 20, 8), S.attention(2, 1, 16)], [None] * 3, (0, 3, 2), width=65, vocab=90),
    "tensor_core_sizes": S.config([S.parallel(4, 2, 64, 64, 70, 32, mem=(2, 64, 64)), S.attention(2, 1, 128, 0.2), S.parallel(2, 1, 128, 128, 100, 128, mem=(1, 128, 128), scale=0.1)],
                                  [S.moe(9, 3, 64), S.moe(4, 2, 72), None], (1, 3, 2), width=128, vocab=128),
    "once": S.config([S.parallel(3, 1, 16, 8, 0, 0), S.attention(6, 2, 13), S.parallel(mem=(3, 10, 7))], [S.moe(2, 1, 16), None, S.moe(5, 5, 24)], (0, 2, 1), width=96, vocab=77),
    "last_layer_loops": S.config([S.attention(), S.parallel(chunk=33)], [None, S.moe(4, 2, 16)], (1, 2, 4), width=64, vocab=64),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_portions_and_decode_match_the_plain_model(name, dtype):
    cfg = CONFIGS[name]
    W = S.weights(cfg, 11, dtype == BF16)
    ids = toks(140, cfg["vocab"], 1)
    layers = []
    ref = P.forward(cfg, W, ids, torch.float32, layers)
    m = build(cfg, W, dtype)
    tol = model_tol(cfg, W, dtype, ids)
    check(run_portions(m, ids, [140], slot=2, tab=[4, 9, 6]), ref, tol, dtype)
    for cuts in ([2], [5, 1, 2, 40], [63, 2, 64]):
        check(run_portions(m, ids, cuts, slot=1, tab=[7, 3, 5]), ref, tol, dtype)
    m.zero_state(3)
    check(run_decode(m, ids[:70], slot=3, tab=[1, 2]), ref[:70], tol, dtype)
    # prompt, then single tokens through the graph
    m.zero_state(0)
    m.forward_batch([(ids[:61], 0, 0, [11, 12, 13])], [[]])
    check(run_decode(m, ids, slot=0, tab=[11, 12, 13], start=61), ref[61:], tol, dtype)
    # the residual after every run of a layer
    seen = []
    m.layer_hook = lambda i, x: seen.append(x.float().cpu().clone())
    m.zero_state(2)
    m.forward_batch([(ids, 0, 2, [4, 9, 6])], [[139]])
    assert len(seen) == len(layers) and all(row_error(a, b) < (1e-5 if dtype == F32 else 0.05) for a, b in zip(seen, layers))


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_match_each_sequence_alone(dtype):
    cfg, W = S.ALL, S.weights(S.ALL, 12, dtype == BF16)
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
    check(torch.cat([torch.cat(g) for g in got]), torch.cat(alone), model_tol(cfg, W, dtype, seqs[-1]), dtype)


@pytest.mark.parametrize("rows", [3, 8, 11, 40])
def test_decode_buckets_match_the_plain_model(rows):
    """Batches of single tokens of unequal sequences, padded to a bucket; above 8 rows on the GEMM path."""
    cfg, W = S.ALL, S.weights(S.ALL, 13, True)
    m = build(cfg, W, BF16, slots=rows, blocks=4 * rows + 1)
    lens = [3 + 5 * i for i in range(rows)]
    seqs = [toks(n + 5, cfg["vocab"], 50 + n) for n in lens]
    tabs = [[1 + 4 * i + k for k in range(4)] for i in range(rows)]
    for i in range(rows):
        m.forward_batch([(seqs[i][:lens[i]], 0, i, tabs[i])], [[]])
    M, got = m.bucket_for(rows), []
    for k in range(5):
        m.set_rows(M, [seqs[i][lens[i] + k] for i in range(rows)], [lens[i] + k for i in range(rows)], list(range(rows)), tabs)
        got.append(m.decode(M)[1][:rows].clone())
    ids = range(0, rows, 1 + rows // 4)
    out = torch.cat([torch.stack([g[i] for g in got]) for i in ids])
    ref = torch.cat([plain_logits(cfg, W, seqs[i])[lens[i]:] for i in ids])
    check(out, ref, model_tol(cfg, W, BF16, seqs[-1]), BF16)


def test_long_decode_in_32_bit():
    cfg, W = S.ALL, S.weights(S.ALL, 14)
    m = build(cfg, W, F32)
    ids = toks(330, cfg["vocab"], 9)
    m.forward_batch([(ids[:10], 0, 0, table(330))], [[]])
    got = run_decode(m, ids, start=10)
    assert rel(got[-40:], plain_logits(cfg, W, ids)[-40:]) < 2e-4


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_trace_replay_reuses_pages_and_slots(dtype):
    """Requests come and go through a pool just large enough; every wanted position equals the plain model."""
    from coffin_b200.engine.replay import TraceReplayer, pool_blocks
    cfg, W = S.ALL, S.weights(S.ALL, 15, dtype == BF16)
    m = build(cfg, W, dtype, slots=4, blocks=pool_blocks(384), max_seq=384)
    rep = TraceReplayer(m)
    r = random.Random(3)
    seqs = {f"q{i}": toks(n, cfg["vocab"], 70 + i) for i, n in enumerate((100, 60, 64, 20, 65, 128, 12, 90))}
    todo, at, live = list(seqs), {}, []
    got = {k: [] for k in seqs}
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
        i = 0
        for e in entries:
            got[e["id"]].append(out[i:i + len(e["want"])])
            i += len(e["want"])
        live = [k for k in live if k not in end]
    # one comparison over all rows: a quantile over the few rows of a short sequence would be one row
    out, ref = (torch.cat(v) for v in ([torch.cat(p) for p in got.values()], [plain_logits(cfg, W, seqs[k]) for k in got]))
    check(out, ref, model_tol(cfg, W, dtype, seqs["q5"]), dtype)
    assert all(rel(torch.cat(p), plain_logits(cfg, W, seqs[k])) < (1e-4 if dtype == F32 else 0.1) for k, p in got.items())
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
    cfg, W = S.ALL, S.weights(S.ALL, 16)
    m = build(cfg, W, F32, slots=3, blocks=24, max_seq=256)
    eng = LLMEngine(m, EngineConfig(max_seq=256, max_num_seqs=3, chunk=48, prefill_quantum=48, max_num_batched_tokens=64,
                                    mixed_batch=mixed, snapshot_interval=64))
    prompts = [toks(n, cfg["vocab"], 90 + n) for n in (70, 9, 40, 130, 3)]
    params = SamplingParams(max_tokens=8, ignore_eos=True)
    seqs = eng.generate(prompts, params)
    prompts.append(prompts[3][:128] + [7])                     # shares a cached prefix: pages by reference, states restored
    seqs += eng.generate(prompts[-1:], params)
    assert (eng.runner.n_mixed_steps > 0) == mixed and eng.runner.n_cached_tokens > 0 and not m.stateless
    for s, p in zip(seqs, prompts):
        assert s.output == plain_greedy(cfg, W, p, 8)


def test_copied_pages_hold_the_factors_of_their_keys():
    """A page copied to another block gives the same logits: keys, values and the keys' factors move together."""
    cfg = S.config([S.attention(4, 2, 24), S.attention(6, 3, 64)], [None, None])
    W, ids = S.weights(cfg, 20), toks(100, 96, 3)
    for dtype in (F32, BF16):
        m = build(cfg, W, dtype)
        assert m.stateless
        m.forward_batch([(ids[:90], 0, 0, [3, 4])], [[]])
        for src, dst in ((3, 8), (4, 6)):
            m.copy_block(src, dst)
        a = m.forward_batch([(ids[90:], 90, 0, [3, 4])], [list(range(10))]).clone()
        b = m.forward_batch([(ids[90:], 90, 1, [8, 6])], [list(range(10))])
        assert torch.equal(a, b)


def test_llm_entry_point_generates_the_engines_tokens(tmp_path):
    from coffin_b200.config import load_config
    from coffin_b200.engine.llm import LLM
    from coffin_b200.models.nodutar.config import NodutarConfig
    from coffin_b200.weights.init import save_checkpoint
    cfg, W = S.ALL, S.weights(S.ALL, 17)
    save_checkpoint(NodutarConfig.from_hf(cfg), W, tmp_path)
    assert load_config(tmp_path).layer_types[:2] == ("attention", "parallel")
    llm = LLM.from_pretrained(tmp_path, max_seq=256, dtype=torch.float32)
    p = toks(50, cfg["vocab"], 4)
    out = llm.generate(p, max_new_tokens=12)
    assert out.tokens == plain_greedy(cfg, W, p, 12)
    first = llm.device_prefill(torch.tensor(p).cuda())
    assert [int(first[0])] + llm.device_decode(first, 11).tolist() == out.tokens


def test_bad_batches_stop_on_the_host():
    m = build(S.ALL, S.weights(S.ALL, 18), BF16, slots=2, blocks=4)
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
    from coffin_b200.models.nodutar.config import NodutarConfig
    from coffin_b200.serving.transport import call, serve
    from coffin_b200.weights.init import save_checkpoint
    cfg = S.config([S.parallel(), S.attention(), S.parallel(4, 2, 24, 40, 33, 8)], [S.moe(3, 3, 16), None, S.moe(4, 4, 16)], (0, 2, 2), vocab=300)
    W = S.weights(cfg, 19, True)
    save_checkpoint(NodutarConfig.from_hf(cfg), W, tmp_path / "model")
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

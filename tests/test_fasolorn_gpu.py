"""Fasolorn on the device against the plain restatement of its equations (``plain_fasolorn.py``)."""
import random

import pytest
import torch

import fasolorn_cases as S
import plain_fasolorn as P
from test_zufilorn_gpu import rel, run_decode, run_portions, table, toks

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
# rms of the error over the rms of the value: 32-bit mode, serving mode
TOL = {F32: 2e-5, BF16: 2e-2}


def build(cfg, W, dtype=F32, slots=4, blocks=40, max_seq=640, **kw):
    from coffin_b200.models import build_model
    from coffin_b200.models.fasolorn.config import FasolornConfig
    return build_model(FasolornConfig.from_hf(cfg), W, device="cuda", dtype=dtype, num_slots=slots, num_blocks=blocks, max_seq=max_seq, **kw)


@torch.no_grad()
def plain_logits(cfg, W, ids):
    return P.forward(cfg, W, ids, torch.float32)


def row_error(got, ref, q=0.9):
    """Quantile over the rows of the row's error: a choice of experts that falls differently after rounding spoils one row."""
    got, ref = got.double().cpu(), ref.double().cpu()
    return float(((got - ref).pow(2).mean(-1) / ref.pow(2).mean()).sqrt().quantile(q))


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


def check(got, ref, tol, dtype):
    if dtype == F32:
        assert rel(got, ref) < tol, rel(got, ref)
    else:
        assert row_error(got, ref) < tol, (row_error(got, ref), tol)


def randn(seed, *s):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


# ------------------------------------------------------------------ the residual
@pytest.mark.parametrize("T,W", [(1, 64), (1, 2560), (5, 72), (3, 50), (200, 512), (2, 33), (1, 1030), (2, 6000), (1, 4098), (1, 9001)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_residual_step(T, W, dtype):
    from coffin_b200.ops import mixers as X
    W8 = (W + 7) // 8 * 8
    x, gain = randn(1, T, W).cuda() * 3, randn(3, W).cuda()
    y, h = torch.zeros(T, W8, dtype=dtype, device="cuda"), torch.zeros(T, W8, dtype=dtype, device="cuda")
    y[:, :W] = randn(2, T, W).to(dtype)
    tol, new, keep = (2e-6 if dtype == F32 else 4e-3), x.double() + y[:, :W].double(), x.clone()
    norm = lambda u: P.rms(u, gain.double(), 1e-3)
    X.residual_step(x, h, gain=gain, eps=1e-3)                                              # nothing to add
    assert torch.equal(x, keep) and rel(h[:, :W], norm(keep.double())) < tol
    X.residual_step(x, h, gain=gain, y=y, eps=1e-3, store=False)
    assert torch.equal(x, keep) and rel(h[:, :W], norm(new)) < tol
    rows = torch.arange(T - 1, -1, -1, dtype=torch.int32, device="cuda")[:2]
    h2 = torch.zeros(rows.numel(), W8, dtype=dtype, device="cuda")
    X.residual_step(x, h2, gain=gain, y=y, rows=rows, store=False, eps=1e-3)
    assert rel(h2[:, :W], norm(new)[rows.long()]) < tol
    X.residual_step(x, h, gain=gain, y=y, eps=1e-3)
    assert rel(x, new) < 1e-6 and rel(h[:, :W], norm(new)) < tol
    X.residual_step(x, None, y=y)                                                           # write-back alone
    assert rel(x, new + y[:, :W].double()) < 1e-6
    # expert rows: slots without a row, a multiple of the input that the norm overwrites
    k = 5
    ys = torch.zeros(T * k + 3, W8, dtype=dtype, device="cuda")
    ys[:, :W] = randn(5, T * k + 3, W).to(dtype)
    pos = torch.randperm(T * k + 3, generator=torch.Generator().manual_seed(1))[:T * k].view(T, k).int()
    pos[:, 2] = -1
    w, idw = randn(6, T, k), randn(7, T, 1)
    idw[0] = 0.0
    hin = h.clone()
    add = sum(w[:, j, None].double() * ys[pos[:, j].long().clamp(min=0).cuda(), :W].double().cpu() for j in (0, 1, 3, 4))
    before = x.double().cpu()
    X.residual_step(x, h, gain=gain, experts=(ys, pos.cuda(), w.cuda(), idw.cuda(), h), eps=1e-3)
    want = before + add + idw.double() * hin[:, :W].double().cpu()
    assert rel(x, want) < 1e-6 and rel(h[:, :W], P.rms(want, gain.double().cpu(), 1e-3)) < tol
    assert (h[:, W:] == 0).all()
    X.residual_step(x, None, experts=(ys, pos.cuda(), w.cuda(), None, None))
    assert rel(x, want + add) < 1e-6


def test_embedding_is_scaled():
    from coffin_b200.ops import mixers as X
    E, tok = randn(5, 30, 44).bfloat16().cuda(), torch.tensor([3, 29, 0, 3]).cuda()
    for e in (E, E.float()):
        assert torch.equal(X.residual_embed(e, tok, torch.zeros(4, 44, device="cuda"), 5.5), E[tok].float() * 5.5)


# ------------------------------------------------------------------ routing and experts
def slots_of(r, T):
    i32 = lambda *s: torch.full(s, -7, dtype=torch.int32, device="cuda")
    return i32(T, r.slots), torch.full((T, r.slots), 9.0, device="cuda"), torch.full((T, 1), 9.0, device="cuda")


@pytest.mark.parametrize("E,ident,top,always", [(7, 3, 3, 2), (4, 0, 1, 0), (5, 1, 6, 1), (128, 16, 8, 1), (300, 212, 32, 4), (1, 1, 1, 0)])
@pytest.mark.parametrize("T", [1, 8, 33, 64, 100])
def test_routing(E, ident, top, always, T):
    from coffin_b200.ops import routed as R
    r, n = R.Router(E, ident, top, 1.7, always), E + ident
    z, corr = randn(1, T, n) * 2, randn(2, n) * 0.2
    zd = torch.zeros(T, n + 5, device="cuda")
    zd[:, :n] = z
    idx, w, idw = slots_of(r, T)
    positions = torch.arange(T, dtype=torch.int32)
    positions[T // 2] = -1                                           # padding: no slots
    ref_i, ref_w = P.route(z.double(), corr.double(), {"top": top, "scale": 1.7})
    lists = [None]
    if T <= R.UNIT_ROWS:
        lists.append(torch.full((R.meta_size(r, T),), -5, dtype=torch.int32, device="cuda"))
    for meta in lists:
        for pos in (None, positions.cuda()):
            if meta is None:
                R.route(r, zd, corr.cuda(), pos, idx, w, idw)
            else:
                d = R.route_units(r, zd, corr.cuda(), pos, idx, w, idw, meta)
            gi, gw, gid = idx.cpu(), w.cpu().double(), idw.cpu().double()
            for t in range(T):
                if pos is not None and t == T // 2:
                    assert (gi[t] == -1).all() and (gw[t] == 0).all() and gid[t] == 0
                    continue
                want = {int(i): float(v) for i, v in zip(ref_i[t], ref_w[t])}
                got = {int(i): float(v) for i, v in zip(gi[t, :top], gw[t, :top]) if i >= 0}
                assert set(got) == {i for i in want if i < E}
                assert all(abs(got[i] - want[i]) < 1e-5 for i in got)
                assert abs(float(gid[t]) - sum(v for i, v in want.items() if i >= E)) < 1e-5
                assert gi[t, top:].tolist() == [E + j for j in range(always)] and (gw[t, top:] == 1).all()
            if meta is None:
                continue
            # the units cover every slot once, in rows of its expert, at most 8 at a time
            c = int(d["count"])
            flat, p, src = idx.cpu().view(-1), d["pos"].cpu(), d["src_tok"].cpu()
            owner = {}
            for k in range(c):
                r0, rn, e = int(d["row0"][k]), int(d["rows"][k]), int(d["expert"][k])
                assert 1 <= rn <= 8
                owner.update({row: e for row in range(r0, r0 + rn)})
            assert sorted(owner) == sorted(int(v) for v in p if v >= 0) == list(range(int((flat >= 0).sum())))
            for s in range(T * r.slots):
                if flat[s] < 0:
                    assert p[s] == -1
                else:
                    assert owner[int(p[s])] == int(flat[s]) and int(src[p[s]]) == s // r.slots
            assert c <= d["max_tiles"] and sum(-(-int(v) // 8) for v in torch.bincount(flat[flat >= 0], minlength=1)) == c


def test_correction_decides_the_choice_but_not_the_weights():
    from coffin_b200.ops import routed as R
    r = R.Router(4, 1, 2, 1.0)
    z = torch.tensor([[3.0, 2.0, 0.0, -1.0, 1.0]]).cuda()
    s = torch.softmax(z[0].cpu().double(), 0)
    for corr, chosen in (([0.0] * 5, (0, 1)), ([0.0, 0.0, 0.0, 5.0, 0.0], (3, 0)), ([-2.0, 0.0, 0.0, 0.0, 1.0], (4, 1)), ([-9.0] * 5, (0, 1))):
        idx, w, idw = slots_of(r, 1)
        R.route(r, z, torch.tensor(corr).cuda(), None, idx, w, idw)
        tot = s[list(chosen)].sum()
        for k, e in enumerate(chosen):
            assert int(idx[0, k]) == (e if e < 4 else -1)
            got = float(w[0, k]) if e < 4 else float(idw[0, 0])
            assert abs(got - float(s[e] / tot)) < 1e-6
        assert 4 in chosen or float(idw[0, 0]) == 0


@pytest.mark.parametrize("N,Kd", [(56, 72), (520, 2048), (2048, 520), (16, 8), (40, 1032)])
@pytest.mark.parametrize("T,top", [(1, 3), (8, 3), (40, 2), (64, 1)])
def test_unit_products(N, Kd, T, top):
    from coffin_b200.ops import kernels as K
    from coffin_b200.ops import routed as R
    r = R.Router(9, 2, top, 1.0, 1)
    z = randn(3, T, 11) * 3
    W, x = (randn(1, 10, N, Kd) * Kd ** -0.5).bfloat16(), randn(2, T, Kd).bfloat16()
    idx, w, idw = slots_of(r, T)
    meta = torch.zeros(R.meta_size(r, T), dtype=torch.int32, device="cuda")
    d = R.route_units(r, z.cuda(), torch.zeros(11).cuda(), None, idx, w, idw, meta)
    flat, pos = idx.cpu().view(-1).long(), d["pos"].cpu().long()
    keep = flat >= 0
    src = torch.arange(T).repeat_interleave(r.slots)[keep]
    ref = torch.einsum("snk,sk->sn", W.double()[flat[keep]], x.double()[src])
    for dtype, tol in ((F32, 2e-6), (BF16, 4e-3)):
        out = torch.full((T * r.slots, N), 3.0, dtype=dtype, device="cuda")
        Wd, xd = W.to(dtype).cuda(), x.to(dtype).cuda()
        R.unit_linear(Wd, xd, out, d, rows=T, gather=True)
        assert rel(out[pos[keep]], ref) < tol
        R.unit_linear(Wd, xd, out, d, rows=T, gather=True, relu2=True)
        assert rel(out[pos[keep]], torch.relu(ref) ** 2) < tol
        rows = torch.zeros(T * r.slots, Kd, dtype=dtype, device="cuda")
        rows[pos[keep]] = xd[src]
        R.unit_linear(Wd, rows, out, d, rows=T, gather=False)
        assert rel(out[pos[keep]], ref) < tol
        assert (out[int(keep.sum()):] == 3).all()
    K.check_status()


MOE = {"all": S.moe(), "no_identity": S.moe(5, 0, 2), "no_shared": S.moe(6, 2, 2, 24, 0), "one_of_many": S.moe(30, 4, 1, 16, 16), "all_of_them": S.moe(3, 2, 5, 32, 100),
       "narrow_shared": S.moe(4, 1, 2, 48, 8), "mostly_identity": S.moe(2, 9, 3, 16, 24), "large": S.moe(6, 2, 2, 264, 520), "odd": S.moe(5, 1, 2, 13, 29, 0.3), "wide_shared": S.moe(9, 2, 3, 8, 333)}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(MOE))
@pytest.mark.parametrize("width", [72, 65])
def test_routed_feed_forward(name, dtype, width):
    """Few rows, units, grouped GEMM: every count of rows gives the plain result."""
    from coffin_b200.ops import mixers as X
    cfg = S.config([S.latent()], [MOE[name]], width=width)
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


def test_experts_of_one_token_batch_match_the_sorted_path():
    """All tokens to the same experts, and every token to another: full units, single rows, uneven tiles."""
    from coffin_b200.ops import mixers as X
    mlp = S.moe(12, 1, 2, 16, 16)
    cfg = S.config([S.latent()], [mlp])
    W = S.weights(cfg, 7)
    W["l0.mlp.router"] = torch.zeros(13, 72).bfloat16()
    for e in range(13):
        W["l0.mlp.router"][e, e] = 4.0
    m = build(cfg, W, BF16)
    ff = {k[7:]: v.double() for k, v in W.items() if k.startswith("l0.mlp.")}
    for T in (64, 150):
        for pattern in ("same", "spread"):
            h = randn(8, T, 72) * 0.3
            h[:, :13] = 0.0
            pick = torch.zeros(T, dtype=torch.long) if pattern == "same" else torch.arange(T) % 12
            h[torch.arange(T), pick], h[torch.arange(T), (pick + 1) % 13] = 2.0, 1.0
            h = h.bfloat16()
            b, _, _ = m.make_batch([([0] * T, 0, 0, table(T))])
            hb = m.buf("h", T, 72)
            hb.copy_(h)
            x = torch.zeros(T, 72, device="cuda")
            X.residual_step(x, None, **m.layers[0].routed.run(m, b, hb))
            assert rel(x, P.experts(h.double(), ff, mlp)) < TOL[BF16], (T, pattern)


# ------------------------------------------------------------------ mixers alone
MIX = {
    "attention": S.attention(), "one_head": S.attention(1, 1, 8, 8, 3, 4), "no_window": S.attention(window=0), "window_1": S.attention(window=1),
    "window_64": S.attention(window=64), "window_65": S.attention(window=65), "window_63": S.attention(4, 4, 16, 16, 63), "window_far": S.attention(window=500),
    "no_rotation": S.attention(rot=0), "all_rotated": S.attention(4, 2, 24, 16, 40, 24), "groups_of_12": S.attention(24, 2, 16, 24, 50, 8), "square": S.attention(3, 3, 64, 64, 30, 32),
    "64_128": S.attention(4, 2, 64, 128, 50, 64), "128": S.attention(4, 1, 128, 128, 90, 64, scale=0.1), "192_64": S.attention(2, 2, 192, 64, 40, 10, scale=0.07),
    "256": S.attention(2, 1, 256, 256, 70, 64, scale=0.06), "odd": S.attention(3, 3, 7, 10, 20, 6), "odd_values": S.attention(4, 2, 16, 13, 33, 16), "large_values": S.attention(2, 1, 32, 300, 40, 8),
    "latent": S.latent(), "latent_no_window": S.latent(window=0), "latent_window_1": S.latent(window=1), "latent_window_64": S.latent(window=64),
    "latent_one_head": S.latent(1, 8, 4, 8, 16, 9), "latent_many": S.latent(20, 16, 8, 16, 48, 70), "latent_32": S.latent(32, 32, 32, 32, 64, 33),
    "latent_wide": S.latent(3, 128, 64, 128, 512, 100, scale=192 ** -0.5), "latent_odd": S.latent(3, 11, 6, 13, 45, 30), "latent_256": S.latent(2, 192, 64, 256, 256, 65),
    "latent_long_head": S.latent(2, 288, 16, 48, 64, 50, scale=0.05), "latent_large_rank": S.latent(2, 16, 8, 24, 600, 47),
}
EPS = 2e-5


def plain_mixer(layer, W, h, first=None, i=0, win=None):
    """``win``: another window (a mistake planted in the equations)."""
    mix = {k[7:]: v.double() for k, v in W.items() if k.startswith(f"l{i}.mix.")}
    m = layer["mixer"] if win is None else dict(layer["mixer"], mask={"size": win})
    if layer["type"] == "attention":
        return P.attention(h.double(), mix, m, first)[0]
    return P.latent_attention(h.double(), mix, m, EPS)


def run_mixer(m, mixers, hs, cuts, slot=1, tab=None):
    """The given mixers on rows ``hs`` (one input each), cut into portions; their outputs."""
    T = hs[0].shape[0]
    tab = tab or table(T, first=2, step=2)
    outs, at, k = [[] for _ in mixers], 0, 0
    while at < T:
        n = min(cuts[k % len(cuts)], T - at)
        k += 1
        b, _, _ = m.make_batch([([0] * n, at, slot, tab)])
        for o, mix, h in zip(outs, mixers, hs):
            hb = m.buf("h", n, (h.shape[1] + 7) // 8 * 8)
            hb[:, :h.shape[1]].copy_(h[at:at + n])
            act = mix.run(m, b, hb)
            o.append(m.linear(mix.w_out, act, m.buf("y", n, mix.w_out.shape[0]))[:, :h.shape[1]].float().clone())
        at += n
    return [torch.cat(o) for o in outs]


def mixer_pair(layer, dtype, T, cuts=None, seed=3, h=None, W=None):
    """(device, plain) outputs of one mixer on the same rows, cut into portions."""
    cfg = S.config([layer], [None], width=64)
    W = W or S.weights(cfg, seed)
    m = build(cfg, W, dtype)
    h = randn(seed + 1, T, 64).bfloat16() if h is None else h
    got, = run_mixer(m, [m.layers[0].mixer], [h], cuts or [T])
    m.check_status()
    return got, plain_mixer(layer, W, h)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(MIX))
def test_mixer_alone(name, dtype):
    for cuts in (None, [1]):
        got, ref = mixer_pair(MIX[name], dtype, 150, cuts)
        assert rel(got, ref) < TOL[dtype], (cuts, rel(got, ref))
        assert rel(got[:3], ref[:3]) < 2 * TOL[dtype]               # the first tokens: one key, two, three


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["attention", "128", "odd", "groups_of_12", "window_65", "latent", "latent_wide", "latent_odd", "latent_long_head"])
@pytest.mark.parametrize("cuts", [[2], [3, 1, 17], [24, 25], [64], [63, 2, 65], [130, 3]])
def test_mixer_in_portions(name, dtype, cuts):
    got, ref = mixer_pair(MIX[name], dtype, 200, cuts)
    assert rel(got, ref) < TOL[dtype], rel(got, ref)
    worst = max(rel(got[i:i + 1], ref[i:i + 1]) for i in range(200))
    assert worst < 8 * TOL[dtype], worst


@pytest.mark.parametrize("layer", [S.attention(4, 2, 64, 64, 100, 32, scale=0.6), S.attention(2, 1, 128, 256, 129, 128, scale=0.4), S.attention(2, 2, 64, 128, 64, 8, scale=0.6),
                                   S.attention(4, 1, 256, 64, 300, 64, scale=0.3), S.latent(3, 128, 64, 128, 96, 70, scale=0.25), S.latent(3, 64, 64, 200, 96, 200, scale=0.3)])
def test_prompt_attention_kernels_agree(layer):
    """tcgen05, mma.sync and the plain equations on prompts and long portions; peaky scores, so that the reference maximum is
    raised again and again, and windows that leave whole pages of a tile to some of its rows."""
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


def test_absorbed_and_expanded_forms_agree(monkeypatch):
    from coffin_b200.models import latent as M
    layer = S.latent(4, 32, 16, 48, 96, 60, scale=0.5)
    a, ref = mixer_pair(layer, BF16, 250, [70, 180])
    monkeypatch.setattr(M, "ABSORB_ROWS", 10 ** 9)
    b, _ = mixer_pair(layer, BF16, 250, [70, 180])
    assert rel(a, ref) < TOL[BF16] and rel(b, ref) < TOL[BF16] and rel(a, b) < TOL[BF16]


@pytest.mark.parametrize("nsplit", [1, 2, 3, 7])
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_key_splits_of_a_window(kind, nsplit, monkeypatch):
    """More splits than pages, splits that start in the middle of the walk, windows that start in the middle of a page."""
    from coffin_b200.ops import mixers as X
    for cls in (X.AttnMaps, X.LatentAttn):
        monkeypatch.setattr(cls, "decode_splits", lambda self, rows: nsplit)
    for win in (1, 63, 64, 65, 130, 200):
        layer = S.attention(4, 2, 16, 24, win, 8) if kind == "attention" else S.latent(4, 16, 8, 24, 40, win)
        got, ref = mixer_pair(layer, BF16, 230, [190, 1])
        assert rel(got[190:], ref[190:]) < TOL[BF16], win


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_values_of_the_first_layer_are_mixed_in(dtype):
    """Three attention layers on inputs of their own: the second takes its share of the first one's values, the third (without
    mixing) does not, and what a page holds is the mixture."""
    ls = [S.attention(4, 2, 16, 24, 40, 8), S.attention(6, 3, 24, 16, 70, 12), S.attention(2, 1, 16, 24, 30, 8, v_mix=False)]
    cfg = S.config(ls, [None] * 3, width=64)
    W = S.weights(cfg, 4)
    W["l1.mix.vmix"] = torch.tensor(0.7).bfloat16()
    m = build(cfg, W, dtype)
    hs = [randn(20 + i, 150, 64).bfloat16() for i in range(3)]
    own = hs[0].double() @ W["l0.mix.v"].double().T
    refs = [plain_mixer(ls[0], W, hs[0], None, 0), plain_mixer(ls[1], W, hs[1], own, 1), plain_mixer(ls[2], W, hs[2], None, 2)]
    for cuts in ([150], [70, 1, 3, 20], [1]):
        for got, ref in zip(run_mixer(m, [l.mixer for l in m.layers], hs, cuts), refs):
            assert rel(got, ref) < TOL[dtype], (cuts, rel(got, ref))
    assert rel(plain_mixer(ls[1], W, hs[1], None, 1), refs[1]) > 0.2


def test_sinks_take_their_share():
    """A sink far above, near and far below the scores; leaving it out changes the output where it matters."""
    layer = S.attention(3, 1, 16, 16, 20, 8)
    cfg = S.config([layer], [None], width=64)
    W = S.weights(cfg, 5)
    for sink in (9.0, 2.0, -30.0):
        W["l0.mix.sink"] = torch.tensor([sink, sink - 1, sink + 1]).bfloat16()
        for dtype in (F32, BF16):
            for cuts in ([100], [1], [60, 1, 7]):
                got, ref = mixer_pair(layer, dtype, 100, cuts, W=W)
                assert rel(got, ref) < TOL[dtype], (sink, cuts)
        blind = dict(W, **{"l0.mix.sink": torch.full((3,), -1e4)})
        off = rel(plain_mixer(layer, blind, randn(4, 100, 64).bfloat16()), ref)
        assert off > 0.1 if sink > 0 else off < 1e-3
    W["l0.mix.sink"] = torch.tensor([120.0, 300.0, -300.0]).bfloat16()      # far outside the range of an exponential
    for cuts in ([100], [1]):
        got, ref = mixer_pair(layer, BF16, 100, cuts, W=W)
        assert torch.isfinite(got).all() and rel(got, ref) < TOL[BF16]


def standout(kind, win):
    """A layer and weights with which a key whose row has a mark (column 63) stands out for every query (column 62 of all rows)."""
    layer = S.attention(4, 2, 16, 24, win, 8, scale=0.5) if kind == "attention" else S.latent(4, 16, 8, 24, 40, win, scale=0.5, base=1e7)
    cfg = S.config([layer], [None], width=64)
    W = S.weights(cfg, 8)
    if kind == "attention":
        q, k = W["l0.mix.q"].float() * 0.2, W["l0.mix.k"].float()
        q[:, 62:], k[:, 62:] = 0.0, 0.0
        for hd in range(4):                                        # column 9 of a head does not turn
            q[hd * 16 + 9] = 0.0
            q[hd * 16 + 9, 62] = 4.0
        for g in range(2):
            k[g * 16 + 9] = 0.0
            k[g * 16 + 9, 63] = 4.0
        W["l0.mix.q"], W["l0.mix.k"], W["l0.mix.sink"] = q.bfloat16(), k.bfloat16(), torch.zeros(4).bfloat16()
    else:                                                          # the slow pair of the rotated part, which all heads share
        q, d = W["l0.mix.q"].float() * 0.2, W["l0.mix.dkv"].float()
        q[:, 62:], d[:, 62:] = 0.0, 0.0
        for hd in range(4):
            q[hd * 24 + 16 + 3] = 0.0
            q[hd * 24 + 16 + 3, 62] = 4.0
        d[40 + 3] = 0.0
        d[40 + 3, 63] = 4.0
        W["l0.mix.q"], W["l0.mix.dkv"] = q.bfloat16(), d.bfloat16()
    return layer, W


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("mode", ["prompt", "decode", "portions"])
@pytest.mark.parametrize("kind", ["attention", "latent"])
def test_one_key_decides_until_it_leaves_the_window(kind, mode, dtype):
    """Key ``j`` stands out for every query that sees it.  Windows that end before, at and after page borders; a window one token
    longer or shorter, or a missing key, would show in single rows."""
    T, cuts = 200, {"prompt": [200], "decode": [1], "portions": [37, 2, 64, 1]}[mode]
    for win, js in ((40, (0, 1, 23, 24, 63, 64, 150)), (64, (0, 63, 64, 65)), (65, (0, 62, 63)), (130, (0, 61, 64)), (2, (63, 64))):
        layer, W = standout(kind, win)
        for j in js:
            h = randn(j, T, 64)
            h[:, 62], h[:, 63] = 2.0, 0.0
            h[j, 63] = 2.0
            h = h.bfloat16()
            got, ref = mixer_pair(layer, dtype, T, cuts, h=h, W=W)
            last = min(T, j + win) - 1                             # the last row that sees it
            rows = [i for i in (j, j + 1, last - 1, last, last + 1, last + 2) if j <= i < T]
            for i in rows:
                assert rel(got[i:i + 1], ref[i:i + 1]) < 4 * TOL[dtype], (win, j, i, rel(got[i:i + 1], ref[i:i + 1]))
            assert rel(got, ref) < 2 * TOL[dtype]
            if last + 1 < T:
                longer, shorter = plain_mixer(layer, W, h, win=win + 1), plain_mixer(layer, W, h, win=win - 1)
                assert rel(longer[last + 1], ref[last + 1]) > 20 * TOL[dtype] and rel(shorter[last], ref[last]) > 20 * TOL[dtype], (win, j)


# ------------------------------------------------------------------ whole models
CONFIGS = {
    "all": S.ALL,
    "narrow": S.config([S.latent(2, 8, 4, 8, 24, 16), S.attention(2, 1, 8, 16, 30, 4)], [S.moe(3, 1, 1, 8, 8), S.dense(24)], width=40, vocab=51, scale=1.0),
    "no_ff": S.config([S.attention(4, 2, 8, 8, 20, 8), S.latent(1, 32, 8, 16, 24, 70), S.attention(2, 2, 16, 8, 0, 4)], [None] * 3, width=65, vocab=90),
    "tensor_core_sizes": S.config([S.attention(4, 2, 64, 64, 70, 32), S.latent(2, 64, 64, 64, 128, 65, scale=0.1), S.attention(2, 1, 128, 128, 100, 128, scale=0.09)],
                                  [S.moe(9, 2, 3, 64, 128), S.dense(256), S.moe(4, 1, 2, 72, 200)], width=128, vocab=128, scale=11.0),
    "mixing_starts_late": S.config([S.attention(3, 1, 16, 8, 20, 8, v_mix=False), S.latent(), S.attention(4, 2, 16, 12, 33, 8), S.attention(6, 3, 8, 8, 45, 8)],
                                   [S.moe(2, 6, 3, 16, 0), None, S.dense(40), S.moe(5, 0, 5, 24, 48)], width=96, vocab=77),
}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_portions_and_decode_match_the_plain_model(name, dtype):
    cfg = CONFIGS[name]
    W = S.weights(cfg, 11)
    ids = toks(140, cfg["vocab"], 1)
    layers = []
    ref = P.forward(cfg, W, ids, torch.float32, layers)
    m = build(cfg, W, dtype)
    tol = model_tol(cfg, W, dtype, ids)
    check(run_portions(m, ids, [140], slot=2, tab=[4, 9, 6]), ref, tol, dtype)
    for cuts in ([2], [5, 1, 2, 40], [63, 2, 64]):
        check(run_portions(m, ids, cuts, slot=1, tab=[7, 3, 5]), ref, tol, dtype)
    check(run_decode(m, ids[:70], slot=3, tab=[1, 2]), ref[:70], tol, dtype)
    # prompt, then single tokens through the graph
    m.forward_batch([(ids[:61], 0, 0, [11, 12, 13])], [[]])
    check(run_decode(m, ids, slot=0, tab=[11, 12, 13], start=61), ref[61:], tol, dtype)
    # the residual after every layer
    seen = []
    m.layer_hook = lambda i, x: seen.append(x.float().cpu().clone())
    m.forward_batch([(ids, 0, 2, [4, 9, 6])], [[139]])
    assert len(seen) == len(layers) and all(row_error(a, b) < (1e-5 if dtype == F32 else 0.05) for a, b in zip(seen, layers))


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_match_each_sequence_alone(dtype):
    cfg, W = S.ALL, S.weights(S.ALL, 12)
    m = build(cfg, W, dtype)
    seqs = [toks(n, cfg["vocab"], n) for n in (90, 33, 5, 130)]
    tabs = [[1, 5], [2], [3], [8, 4, 6]]
    alone = [run_portions(m, s, [len(s)], slot=0, tab=t) for s, t in zip(seqs, tabs)]
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
    cfg, W = S.ALL, S.weights(S.ALL, 13)
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
    cfg, W = S.ALL, S.weights(S.ALL, 15)
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
    assert all(rel(torch.cat(p), plain_logits(cfg, W, seqs[k])) < (1e-4 if dtype == F32 else 0.3) for k, p in got.items())
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
    for n, reused in ((128, 128), (90, 64)):                   # cached prefixes: pages by reference, at any page
        before = eng.runner.n_cached_tokens
        prompts.append(prompts[3][:n] + [7])
        seqs += eng.generate(prompts[-1:], params)
        assert eng.runner.n_cached_tokens - before == reused
    assert (eng.runner.n_mixed_steps > 0) == mixed and m.stateless
    for s, p in zip(seqs, prompts):
        assert s.output == plain_greedy(cfg, W, p, 8)


def test_llm_entry_point_generates_the_engines_tokens(tmp_path):
    from coffin_b200.config import load_config
    from coffin_b200.engine.llm import LLM
    from coffin_b200.models.fasolorn.config import FasolornConfig
    from coffin_b200.weights.init import save_checkpoint
    cfg, W = S.ALL, S.weights(S.ALL, 17)
    save_checkpoint(FasolornConfig.from_hf(cfg), W, tmp_path)
    assert load_config(tmp_path).layer_types[:2] == ("attention", "latent_attention")
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
    from coffin_b200.models.fasolorn.config import FasolornConfig
    from coffin_b200.serving.transport import call, serve
    from coffin_b200.weights.init import save_checkpoint
    cfg = S.config([S.attention(), S.latent(), S.attention(4, 2, 24, 40, 33, 8)], [S.dense(), S.dense(64), S.moe(4, 1, 5, 16, 16)], vocab=300)
    W = S.weights(cfg, 19)
    save_checkpoint(FasolornConfig.from_hf(cfg), W, tmp_path / "model")
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

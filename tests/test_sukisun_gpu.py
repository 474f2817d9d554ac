"""Sukisun on the device against the plain restatement of its equations (``plain_sukisun.py``)."""
import random

import pytest
import torch

import plain_sukisun as P
import sukisun_cases as S
from test_zufilorn_gpu import rel, run_decode, run_portions, table, toks

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
# rms of the error over the rms of the value: 32-bit mode, serving mode
TOL = {F32: 2e-5, BF16: 2e-2}


def build(cfg, W, dtype=F32, slots=4, blocks=40, max_seq=640, **kw):
    from coffin_b200.models import build_model
    from coffin_b200.models.sukisun.config import SukisunConfig
    return build_model(SukisunConfig.from_hf(cfg), W, device="cuda", dtype=dtype, num_slots=slots, num_blocks=blocks, max_seq=max_seq, **kw)


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
        errs.append(rel(plain_logits(cfg, near, ids), base))
    return 2 * max(errs)


def randn(seed, *s):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


# ------------------------------------------------------------------ single mechanisms
@pytest.mark.parametrize("T,W,planes", [(1, 64, 2), (1, 2048, 14), (5, 72, 4), (3, 50, 11), (200, 512, 6), (2, 33, 3), (1, 1030, 20), (9, 1536, 9)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_depth_step(T, W, planes, dtype):
    from coffin_b200.ops import mixers as X
    x, y, gain, dwa = randn(1, T, planes, W).cuda() * 3 + 1, randn(2, T, W).to(dtype).cuda(), randn(3, W).cuda(), randn(4, planes).cuda()
    tol, p = (2e-6 if dtype == F32 else 4e-3), planes - 2
    new = x.double()
    new[:, p] += y.double()
    avg = P.depth_average(dwa[:p + 1].double(), [new[:, j] for j in range(p + 1)])
    keep, h = x.clone(), torch.zeros(T, W, dtype=dtype, device="cuda")
    for center in (True, False):
        norm = (lambda u: P.layer_norm(u, gain.double(), 1e-3)) if center else (lambda u: P.rms(u, 1e-3) * gain.double())
        X.depth_step(x, p, h, gain=gain, y=y, weights=dwa[:p + 1], eps=1e-3, store=False, center=center)
        assert torch.equal(x, keep) and rel(h, norm(avg)) < tol
        X.depth_step(x, p, h, gain=gain, y=y, eps=1e-3, store=False, center=center)         # inside a layer: no average
        assert rel(h, norm(new[:, p])) < tol
        X.depth_step(x, p, h, gain=gain, eps=1e-3, center=center)                           # nothing to add
        assert torch.equal(x, keep) and rel(h, norm(keep[:, p].double())) < tol
    rows = torch.arange(T - 1, -1, -1, dtype=torch.int32, device="cuda")[:2]
    h2 = torch.zeros(rows.numel(), W, dtype=dtype, device="cuda")
    X.depth_step(x, p, h2, gain=gain, y=y, weights=dwa[:p + 1], rows=rows, store=False, eps=1e-3)
    assert rel(h2, P.layer_norm(avg, gain.double(), 1e-3)[rows.long()]) < tol
    X.depth_step(x, p, h, gain=gain, y=y, weights=dwa[:p + 1], eps=1e-3)
    assert rel(x[:, p], new[:, p]) < 1e-6 and rel(x[:, p + 1], avg) < 2e-6 and torch.equal(x[:, :p], keep[:, :p])
    X.depth_step(x, p, None, y=y)                                                           # write-back alone
    assert rel(x[:, p], new[:, p] + y.double()) < 1e-6


@pytest.mark.parametrize("T,W", [(1, 64), (1, 2048), (3, 50), (100, 256)])
def test_depth_averages_in_blocks(T, W):
    """Layer by layer through 21 layers: partial sums prepared at the block ends and completed inside the blocks."""
    from coffin_b200.ops import mixers as X
    n = 21
    dwa, gain = randn(1, n, n + 1).cuda(), torch.ones(W, device="cuda")
    x, ref = torch.full((T, n + 2, W), float("nan"), device="cuda"), []
    e = randn(2, T, W).cuda()
    x[:, 0], x[:, 1] = e, e
    h = torch.zeros(T, W, device="cuda")
    ref, cur = [e.double()], e.double()
    for i in range(n):
        y = randn(10 + i, T, W).cuda()
        plan = X.depth_plan(i, n)
        assert plan["first"] in (0, i // X.DEPTH_BLOCK * X.DEPTH_BLOCK + 1) and (plan["prep"] > 0) == (i in (7, 15))
        X.depth_step(x, i + 1, h, gain=gain, y=y, weights=dwa[i:], **plan)
        ref.append(cur + y.double())
        cur = P.depth_average(dwa[i, :i + 2].double(), ref)
        assert rel(x[:, i + 2], cur) < 3e-6 and rel(x[:, i + 1], ref[-1]) < 3e-6 and rel(h, P.layer_norm(cur, gain.double(), 1e-5)) < 3e-6, i
        cur = x[:, i + 2].double()


def test_depth_embed_scales_and_starts_the_first_layer():
    from coffin_b200.ops import mixers as X
    E = randn(5, 30, 44).bfloat16().cuda()
    x = torch.full((4, 3, 44), 7.0, device="cuda")
    tok = torch.tensor([3, 29, 0, 3]).cuda()
    X.depth_embed(E, tok, x, 5.5)
    assert torch.equal(x[:, 0], E[tok].float() * 5.5) and torch.equal(x[:, 1], x[:, 0]) and (x[:, 2] == 7).all()


@pytest.mark.parametrize("M", [1, 3, 8, 9, 40, 130, 300, 600])
@pytest.mark.parametrize("N,Kd", [(88, 72), (512, 264), (1000, 64)])
def test_xielu_in_the_projection(M, N, Kd):
    from coffin_b200.ops import kernels as K
    from coffin_b200.ops import mixers as X
    W, x, act = randn(1, N, Kd).bfloat16(), randn(2, M, Kd).bfloat16() * Kd ** -0.5 * 3, torch.tensor([0.7, -1.1])
    a, b = P.softplus(act.double()).tolist()
    ref = P.xielu(x.double() @ W.double().T, act.double())
    out = torch.zeros(M, N, dtype=BF16, device="cuda")
    X.linear_xielu(W.cuda(), x.cuda(), out, a, 0.5 + b)
    assert rel(out, ref) < 4e-3
    o32 = torch.zeros(M, N, device="cuda")
    X.linear_xielu(W.float().cuda(), x.float().cuda(), o32, a, 0.5 + b)
    assert rel(o32, ref) < 1e-6
    K.check_status()


def test_xielu_branches_meet_at_zero_and_bend_away_from_it():
    from coffin_b200.ops import mixers as X
    z = torch.tensor([-30.0, -4.0, -0.5, -1e-3, -1e-6, 0.0, 1e-6, 1e-3, 0.5, 4.0, 30.0])
    act = torch.tensor([-0.4, 1.2])
    a, b = P.softplus(act.double()).tolist()
    out = torch.zeros(1, z.numel(), device="cuda")
    X.linear_xielu(z[:, None].contiguous().cuda(), torch.ones(1, 1).cuda(), out, a, 0.5 + b)
    assert torch.allclose(out[0].cpu().double(), P.xielu(z.double(), act.double()), rtol=1e-6, atol=1e-9)


def test_rotary_angles_stay_exact_far_out():
    from coffin_b200.ops import mixers as X
    pos = torch.tensor([0, 1, 63, 1000, 54321, 1 << 20], dtype=torch.int32).cuda()
    turns = X.rope_turns(700.0, 14, "cuda")
    cs = X.rope_rows(pos, turns, torch.zeros(6, 14, device="cuda")).view(6, 7, 2).double().cpu()
    ang = pos.cpu().double()[:, None] * 700.0 ** (-2.0 * torch.arange(7, dtype=torch.float64) / 14)
    assert (cs[..., 0] - ang.cos()).abs().max() < 1e-6 and (cs[..., 1] - ang.sin()).abs().max() < 1e-6


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,rot,dims", [(3, 8, 8), (130, 16, 16), (5, 12, 4), (4, 7, 6)])
def test_rotation_of_head_parts(T, rot, dims, dtype):
    from coffin_b200.ops import mixers as X
    H, hs = 3, 24
    q = randn(6, T, H * hs).to(dtype)
    ref = q.double().view(T, H, hs).clone()
    ref[..., 8:8 + rot] = P.rotate(ref[..., 8:8 + rot], dims, 50.0)
    cs = X.rope_rows(torch.arange(T, dtype=torch.int32).cuda(), X.rope_turns(50.0, dims, "cuda"), torch.zeros(T, dims, device="cuda"))
    d = q.cuda()
    X.rope_heads(d[:, 8:], hs, d[:, 8:], hs, cs, half=dims // 2, rot=rot, H=H)
    assert rel(d, ref.reshape(T, -1)) < (1e-6 if dtype == F32 else 4e-3)
    far = torch.zeros(T, H * 40, dtype=dtype, device="cuda")
    X.rope_heads(q.cuda()[:, 8:], hs, far[:, 5:], 40, cs, half=dims // 2, rot=rot, H=H)
    assert rel(far.view(T, H, 40)[..., 5:5 + rot], ref[..., 8:8 + rot]) < (1e-6 if dtype == F32 else 4e-3)


@pytest.mark.parametrize("T", [1, 7, 12, 30, 64, 70])
@pytest.mark.parametrize("H,N,Kd", [(3, 16, 24), (5, 40, 72), (2, 130, 320), (1, 512, 128), (4, 64, 512)])
def test_per_head_products(T, H, N, Kd):
    from coffin_b200.ops import mixers as X
    w, x, g = randn(1, H, N, Kd), randn(2, T, H * (Kd + 8)), randn(3, T, 8)
    for dtype in (F32, BF16):
        wd, xd = w.to(dtype).cuda(), x.to(dtype).cuda()
        ref = torch.einsum("hnk,thk->thn", wd.double(), xd.double().view(T, H, Kd + 8)[..., :Kd])
        for gate in (None, g.cuda()):
            y = torch.full((T, H * (N + 3)), 5.0, dtype=dtype, device="cuda")
            X.head_linear(wd, xd, Kd + 8, y, N + 3, gate=gate)
            want = ref if gate is None else ref * torch.sigmoid(gate.double())[:, :H, None]
            assert rel(y.view(T, H, N + 3)[..., :N], want) < (2e-6 if dtype == F32 else 4e-3)
            assert (y.view(T, H, N + 3)[..., N:] == 5).all()


@pytest.mark.parametrize("H,cp,rp,nsplit", [(4, 16, 16, 1), (7, 112, 32, 3), (16, 128, 16, 2), (17, 80, 16, 5), (32, 512, 64, 7), (40, 256, 32, 2), (5, 272, 16, 64)])
def test_absorbed_decode_kernel(H, cp, rp, nsplit):
    """Rows of unequal length against scattered pages; one key of every row stands out for one head."""
    from coffin_b200.ops import mixers as X
    LW, lens = cp + rp, (1, 63, 64, 65, 130, 300)
    pool = (randn(1, 40 * 64, LW) * 0.5).bfloat16().cuda()
    order = torch.randperm(39, generator=torch.Generator().manual_seed(2)) + 1
    tabs = torch.stack([order[6 * i:6 * i + 6] if 6 * i + 6 <= 39 else order[:6] for i in range(6)]).int().cuda()
    q = (randn(3, 6, H * LW) * LW ** -0.5).bfloat16().cuda()
    scale, qv = 0.7, q.view(6, H, LW)
    keys = []
    for i, n in enumerate(lens):
        rows = (tabs[i].long()[:, None] * 64 + torch.arange(64, device="cuda")).view(-1)[:n]
        j = (n - 1) // 2                                            # the key that stands out
        qv[i, H - 1] = pool[rows[j]] * 0.3
        keys.append(rows)
    core = X.LatentAttn(H=H, q_rank=8, kv_rank=cp, rot=rp, rot_dims=0, cp=cp, scale=scale, eps=1e-5, pool=pool, norm_q=torch.ones(8).cuda(),
                        norm_c=None)
    assert core.tc
    pos = torch.tensor([n - 1 for n in lens], dtype=torch.int32).cuda()
    po, pm = torch.full((6, H * nsplit * cp), 9.0, device="cuda"), torch.full((6, H * nsplit * 2), 9.0, device="cuda")
    core.absorbed(q, tabs, pos, None, po, pm, nsplit)
    out = torch.zeros(6, H * cp, device="cuda")
    core.merge(po, pm, out, pos, nsplit)
    for i, rows in enumerate(keys):
        k = pool[rows].double()
        ref = torch.softmax(qv[i].double() @ k.T * scale, -1) @ k[:, :cp]
        assert rel(out[i].view(H, cp), ref) < 2e-4, i


@pytest.mark.parametrize("groups,n", [(1, 64), (3, 50), (2, 2560), (8, 24), (1, 13)])
def test_gated_norm(groups, n):
    from coffin_b200.ops import mixers as X
    T, c = 5, groups * n
    y, z, w = randn(1, T, c).cuda() * 4, randn(2, T, c + 8).cuda(), randn(3, c).cuda()
    for dtype in (F32, BF16):
        zd = z.to(dtype)
        u = (y.double() * P.silu(zd.double()[:, :c])).view(T, groups, n)
        act = torch.zeros(T, c + 4, dtype=dtype, device="cuda")
        X.gated_norm(y, zd[:, :c], w, act, groups=groups, n=n, eps=1e-3)
        assert rel(act[:, :c], P.rms(u, 1e-3).view(T, c) * w.double()) < (2e-6 if dtype == F32 else 4e-3)


# ------------------------------------------------------------------ mixers alone
MIX = {
    "mamba": S.mamba(), "mamba_one_group": S.mamba(5, 40, 56, 1, 3, 1), "mamba_groups": S.mamba(6, 16, 16, 6, 2, 6), "mamba_one_tap": S.mamba(2, 8, 24, 1, 1, 2),
    "mamba_64": S.mamba(3, 64, 64, 1, 4, 3), "mamba_128": S.mamba(2, 64, 128, 1, 4, 1), "mamba_256": S.mamba(2, 40, 256, 2, 4, 1),
    "mamba_odd": S.mamba(3, 7, 10, 1, 5, 3), "mamba_wide": S.mamba(1, 136, 72, 1, 6, 1),
    "latent": S.latent(), "latent_one_head": S.latent(1, 8, 4, 8, 16, 8), "latent_many": S.latent(20, 16, 8, 16, 48, 24), "latent_32": S.latent(32, 32, 32, 32, 64, 64),
    "latent_wide": S.latent(3, 128, 64, 128, 512, 192, 192 ** -0.5), "latent_odd": S.latent(3, 11, 6, 13, 45, 19), "latent_big_values": S.latent(2, 48, 16, 200, 136, 40),
    "latent_part": S.latent(4, 16, 24, 24, 64, 32, rot_dims=10), "latent_far_base": S.latent(4, 8, 32, 16, 40, 32, base=5e5), "latent_256": S.latent(2, 192, 64, 256, 256, 64),
    "latent_long_head": S.latent(2, 288, 16, 48, 64, 40, 0.05), "latent_large_rank": S.latent(2, 16, 8, 24, 600, 40),
    "mamba_large_state": S.mamba(2, 16, 320, 1, 4, 1), "mamba_long_conv": S.mamba(2, 16, 16, 2, 20, 1),
}


def plain_mixer(layer, W, h, eps, src=0, hs=None):
    mix = {k[7:]: v.double() for k, v in W.items() if k.startswith("l0.mix.")}
    if layer["type"] == "mamba2":
        return P.mamba2(h.double(), mix, layer["mixer"], eps)
    return P.latent_attention(h.double(), mix, layer["mixer"], eps, P.latents(h.double(), mix, layer["mixer"], eps))


def run_mixer(m, mix, h, cuts, slot=1, tab=None):
    T = h.shape[0]
    tab = tab or table(T, first=2, step=2)
    outs, at, k = [], 0, 0
    while at < T:
        n = min(cuts[k % len(cuts)], T - at)
        k += 1
        b, _, _ = m.make_batch([([0] * n, at, slot, tab)])
        hb = m.buf("h", n, (h.shape[1] + 7) // 8 * 8)
        hb[:, :h.shape[1]].copy_(h[at:at + n])
        act = mix.run(m, b, hb)
        outs.append(m.linear(mix.w_out, act, m.buf("y", n, mix.w_out.shape[0]))[:, :h.shape[1]].float().clone())
        at += n
    return torch.cat(outs)


def mixer_pair(layer, dtype, T, cuts=None, seed=3, h=None, W=None):
    """(device, plain) outputs of one mixer on the same rows, cut into portions."""
    cfg = S.config([layer], width=64, ff=None)
    W = W or S.weights(cfg, seed)
    m = build(cfg, W, dtype)
    h = randn(seed + 1, T, 64).bfloat16() if h is None else h
    m.zero_state(1)
    got = run_mixer(m, m.layers[0].mixer, h, cuts or [T])
    m.check_status()
    return got, plain_mixer(layer, W, h, cfg["norm"]["eps"])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(MIX))
def test_mixer_alone(name, dtype):
    for cuts in (None, [1]):
        got, ref = mixer_pair(MIX[name], dtype, 83, cuts)
        assert rel(got, ref) < TOL[dtype], (cuts, rel(got, ref))
        assert rel(got[:3], ref[:3]) < 2 * TOL[dtype]               # the first tokens: empty state, empty convolution, one key


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mamba", "mamba_128", "mamba_odd", "latent", "latent_wide", "latent_odd", "latent_long_head"])
@pytest.mark.parametrize("cuts", [[2], [3, 1, 17], [24, 25], [64], [63, 2, 65], [130, 3]])
def test_mixer_in_portions(name, dtype, cuts):
    got, ref = mixer_pair(MIX[name], dtype, 200, cuts)
    assert rel(got, ref) < TOL[dtype], rel(got, ref)
    worst = max(rel(got[i:i + 1], ref[i:i + 1]) for i in range(200))
    assert worst < 8 * TOL[dtype], worst


@pytest.mark.parametrize("sizes", [(128, 64, 128), (32, 32, 64), (64, 64, 200), (192, 64, 40), (24, 8, 136)])
def test_prompt_attention_kernels_agree(sizes):
    """tcgen05, mma.sync and the plain equations on prompts and long portions; peaky scores, so that the reference maximum is
    raised again and again."""
    from coffin_b200.ops import kernels as K
    n, r, e = sizes
    layer = S.latent(3, n, r, e, 96, 64, scale=3.0 * (n + r) ** -0.5)
    for cuts in ([333], [130, 203]):
        got, ref = mixer_pair(layer, BF16, 333, cuts, seed=n + e)
        assert rel(got, ref) < 1.5 * TOL[BF16], (cuts, rel(got, ref))
    was, K.ATTN_TC = K.ATTN_TC, False
    try:
        other, _ = mixer_pair(layer, BF16, 333, [130, 203], seed=n + e)
    finally:
        K.ATTN_TC = was
    assert rel(got, other) < 4e-3


def test_absorbed_and_expanded_forms_agree(monkeypatch):
    from coffin_b200.models import latent as M
    layer = S.latent(4, 32, 16, 48, 96, 64, scale=0.5)
    a, ref = mixer_pair(layer, BF16, 150, [70, 80])
    monkeypatch.setattr(M, "ABSORB_ROWS", 10 ** 9)
    b, _ = mixer_pair(layer, BF16, 150, [70, 80])
    assert rel(a, ref) < TOL[BF16] and rel(b, ref) < TOL[BF16] and rel(a, b) < TOL[BF16]


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_borrowed_latents(dtype):
    """A layer with ``kv_from`` attends over the lender's rows (from another input, other head sizes), portion by portion."""
    lend, borrow = S.latent(4, 16, 16, 24, 72, 40), S.latent(6, 24, 16, 40, 72, 56, 0.3, kv_from=0)
    cfg = S.config([lend, borrow], width=64, ff=None)
    W = S.weights(cfg, 4)
    m = build(cfg, W, dtype)
    h0, h1 = randn(1, 120, 64).bfloat16(), randn(2, 120, 64).bfloat16()
    part = lambda i: {k[7:]: v.double() for k, v in W.items() if k.startswith(f"l{i}.mix.")}
    cached = P.latents(h0.double(), part(0), lend["mixer"], 2e-5)
    ref = P.latent_attention(h1.double(), part(1), borrow["mixer"], 2e-5, cached)
    for cuts in ([120], [50, 1, 3], [2]):
        at, k, outs = 0, 0, []
        while at < 120:
            n = min(cuts[k % len(cuts)], 120 - at)
            b, _, _ = m.make_batch([([0] * n, at, 2, [3, 9])])
            hb = m.buf("h", n, 64)
            hb.copy_(h0[at:at + n])
            m.layers[0].mixer.run(m, b, hb)
            hb.copy_(h1[at:at + n])
            mix = m.layers[1].mixer
            outs.append(m.linear(mix.w_out, mix.run(m, b, hb), m.buf("y", n, 64)).float().clone())
            at, k = at + n, k + 1
        assert rel(torch.cat(outs), ref) < TOL[dtype], cuts
    assert m.layers[1].mixer.pools == () and m.layers[1].mixer.pool is m.layers[0].mixer.pool


def test_strong_and_vanishing_decays_stay_finite():
    layer = S.mamba(4, 16, 32, 1, 4, 1)
    cfg = S.config([layer], width=64, ff=None)
    W = S.weights(cfg, 6)
    W["l0.mix.A_log"] = torch.tensor([5.0, 3.0, -6.0, 0.0]).bfloat16()       # decays down to exp(-148 dt) per token
    W["l0.mix.dt_bias"] = torch.tensor([3.0, -4.0, 2.0, -9.0]).bfloat16()
    for dtype in (F32, BF16):
        for cuts in ([150], [70, 1, 9]):
            got, ref = mixer_pair(layer, dtype, 150, cuts, W=W)
            assert torch.isfinite(got).all() and rel(got, ref) < TOL[dtype], rel(got, ref)


def test_state_keeps_a_token_far_back():
    """Decays near one and a token whose value row is far larger than the others: it has to be visible 190 tokens later,
    across chunks, portions and the step kernel."""
    layer = S.mamba(2, 16, 16, 1, 3, 2)
    cfg = S.config([layer], width=64, ff=None)
    W = S.weights(cfg, 7)
    W["l0.mix.A_log"] = torch.full((2,), -7.0).bfloat16()
    w_in = W["l0.mix.in"].float()
    w_in[:, 63] = 0.0
    w_in[32:64, 63] = 20.0                                                   # x rows
    W["l0.mix.in"] = w_in.bfloat16()
    for j in (0, 1, 14, 63, 64, 65, 126):
        h = randn(j, 200, 64)
        h[:, 63] = 0.0
        h[j, 63] = 4.0
        h = h.bfloat16()
        blind = h.clone()
        blind[j, 63] = 0.0
        lost = plain_mixer(layer, W, blind, 2e-5)
        for dtype in (F32, BF16):
            for cuts in ([200], [j + 1, 3, 50], [1]) if dtype == F32 else ([200], [max(1, j), 30]):
                got, ref = mixer_pair(layer, dtype, 200, cuts, h=h, W=W)
                assert rel(got[190:], ref[190:]) < 2 * TOL[dtype]
        assert rel(lost[190:], ref[190:]) > 0.2


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("mode", ["prompt", "decode", "portions"])
@pytest.mark.parametrize("part", ["latent", "rotated"])
def test_one_far_key_decides_the_attention(dtype, mode, part):
    """Key ``j`` is made to stand out for every later query, through the latent or through the shared rotated part (a slow
    pair), at page borders and far back: dropping it, or reading its neighbour, changes the output."""
    m = S.latent(4, 16, 8, 24, 40, 24, scale=0.5, base=1e7)
    cfg = S.config([m], width=64, ff=None)
    W = S.weights(cfg, 8)
    f = {n: W[f"l0.mix.{n}"].float() for n in ("dq", "uq", "dkv", "uk")}
    f["uq"] *= 0.2
    f["dq"][:, 62:] = 0.0
    f["dkv"][:, 62:] = 0.0
    f["dq"][0, :], f["dq"][0, 62] = 0.0, 3.0                       # query latent 0: the same for every token
    q_row, k_row = (0, 0) if part == "latent" else (22, 46)        # head entry of the query; latent 0 or the slow pair's first entry
    for hd in range(4):
        f["uq"][hd * 24 + q_row, :] = 0.0
        f["uq"][hd * 24 + q_row, 0] = 4.0
        if part == "latent":
            f["uk"][hd * 16, :] = 0.0
            f["uk"][hd * 16, 0] = 1.0
    f["dkv"][k_row, :] = 0.0
    f["dkv"][k_row, 63] = 8.0                                      # only the marked row has column 63
    for n, v in f.items():
        W[f"l0.mix.{n}"] = v.bfloat16()
    T, cuts = 200, {"prompt": [200], "decode": [1], "portions": [37, 2, 64]}[mode]
    for j in (0, 1, 62, 63, 64, 65, 127, 128, 191):
        h = randn(j, T, 64)
        h[:, 62], h[:, 63] = 2.0, 0.0
        h[j, 63] = 2.0
        h = h.bfloat16()
        got, ref = mixer_pair(m, dtype, T, cuts, h=h, W=W)
        assert rel(got, ref) < 2 * TOL[dtype], (j, rel(got, ref))
        blind = h.clone()
        blind[j, 63] = 0.0
        assert rel(plain_mixer(m, W, blind, 2e-5)[j + 1:], ref[j + 1:]) > 10 * TOL[dtype], j


# ------------------------------------------------------------------ whole models
CONFIGS = {
    "all": S.ALL,
    "narrow": S.config([S.latent(2, 8, 4, 8, 24, 16), S.mamba(2, 16, 16, 1, 2, 1)], width=40, vocab=51, scale=1.0, ff=24),
    "no_ff": S.config([S.latent(4, 8, 8, 16, 32, 24), S.mamba(1, 32, 8, 1, 4, 1), S.latent(2, 16, 8, 8, 32, 8, kv_from=0)], no_mlp=(0, 1, 2), width=65,
                      vocab=90),
    "sizes_differ": S.config([S.mamba(2, 64, 128, 1, 4, 2), S.latent(8, 64, 64, 64, 256, 96, 0.08), S.latent(3, 16, 8, 24, 48, 40), S.mamba(6, 8, 24, 3, 3, 2),
                              S.latent(18, 32, 64, 32, 256, 64, 0.1, kv_from=1), S.latent(2, 40, 8, 16, 48, 40, kv_from=2)], width=128, ff=200, vocab=128,
                             scale=11.0),
    "deep": S.config([S.latent(2, 8, 4, 8, 24, 16)] + [S.mamba(2, 8, 8, 1, 2, 1), S.latent(2, 8, 4, 8, 24, 16, kv_from=0)] * 9, width=32, vocab=60, ff=24,
                     no_mlp=range(1, 18, 2)),
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
    # the residual after every layer
    seen = []
    m.layer_hook = lambda i, x: seen.append(x.float().cpu().clone())
    m.zero_state(2)
    m.forward_batch([(ids, 0, 2, [4, 9, 6])], [[139]])
    assert len(seen) == len(layers) and all(rel(a, b) < (1e-5 if dtype == F32 else 0.05) for a, b in zip(seen, layers))


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_match_each_sequence_alone(dtype):
    cfg, W = S.ALL, S.weights(S.ALL, 12)
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


@pytest.mark.parametrize("rows", [3, 8, 11, 40])
def test_decode_buckets_match_the_plain_model(rows):
    """Batches of single tokens of unequal sequences, padded to a bucket; above 8 rows on the GEMM path."""
    cfg, W = S.ALL, S.weights(S.ALL, 13)
    m = build(cfg, W, BF16, slots=rows, blocks=4 * rows + 1)
    lens = [3 + 5 * i for i in range(rows)]
    seqs = [toks(n + 5, cfg["vocab"], 50 + n) for n in lens]
    tabs = [[1 + 4 * i + k for k in range(4)] for i in range(rows)]
    for i in range(rows):
        m.zero_state(i)
        m.forward_batch([(seqs[i][:lens[i]], 0, i, tabs[i])], [[]])
    M, got = m.bucket_for(rows), []
    for k in range(5):
        m.set_rows(M, [seqs[i][lens[i] + k] for i in range(rows)], [lens[i] + k for i in range(rows)], list(range(rows)), tabs)
        got.append(m.decode(M)[1][:rows].clone())
    for i in range(0, rows, 1 + rows // 4):
        ref = plain_logits(cfg, W, seqs[i])[lens[i]:]
        assert rel(torch.stack([g[i] for g in got]), ref) < model_tol(cfg, W, BF16, seqs[i]), i


def test_long_decode_in_32_bit():
    cfg, W = S.ALL, S.weights(S.ALL, 14)
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
    cfg, W = S.ALL, S.weights(S.ALL, 15)
    m = build(cfg, W, dtype, slots=4, blocks=pool_blocks(384), max_seq=384)
    rep = TraceReplayer(m)
    r = random.Random(3)
    seqs = {f"q{i}": toks(n, cfg["vocab"], 70 + i) for i, n in enumerate((100, 60, 64, 20, 65, 128, 2, 90))}
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
    cfg, W = S.ALL, S.weights(S.ALL, 16)
    m = build(cfg, W, F32, slots=3, blocks=24, max_seq=256)
    eng = LLMEngine(m, EngineConfig(max_seq=256, max_num_seqs=3, chunk=48, prefill_quantum=48, max_num_batched_tokens=64,
                                    mixed_batch=mixed, snapshot_interval=64))
    prompts = [toks(n, cfg["vocab"], 90 + n) for n in (70, 9, 40, 130, 3)]
    params = SamplingParams(max_tokens=8, ignore_eos=True)
    seqs = eng.generate(prompts, params)
    prompts.append(prompts[3][:128] + [7])                     # shares a cached prefix: pages by reference, states restored
    seqs += eng.generate(prompts[-1:], params)
    assert (eng.runner.n_mixed_steps > 0) == mixed and eng.runner.n_cached_tokens > 0
    for s, p in zip(seqs, prompts):
        assert s.output == plain_greedy(cfg, W, p, 8)


def test_llm_entry_point_generates_the_engines_tokens(tmp_path):
    from coffin_b200.config import load_config
    from coffin_b200.engine.llm import LLM
    from coffin_b200.models.sukisun.config import SukisunConfig
    from coffin_b200.weights.init import save_checkpoint
    cfg, W = S.ALL, S.weights(S.ALL, 17)
    save_checkpoint(SukisunConfig.from_hf(cfg), W, tmp_path)
    assert load_config(tmp_path).layer_types == ("mamba2", "latent_attention") * 2
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
    from coffin_b200.models.sukisun.config import SukisunConfig
    from coffin_b200.serving.transport import call, serve
    from coffin_b200.weights.init import save_checkpoint
    cfg = S.config([S.mamba(), S.latent(), S.latent(3, 16, 16, 24, 72, 40, kv_from=1)], vocab=300)
    W = S.weights(cfg, 19)
    save_checkpoint(SukisunConfig.from_hf(cfg), W, tmp_path / "model")
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

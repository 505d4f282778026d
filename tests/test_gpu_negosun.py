"""Negosun on the GPU against the slow float64 oracle (tests/negosun_oracle.py): each mechanism alone, prompts against
token-by-token decoding, portions, ragged batches, rows given back and used again, far keys in prompts and in decoding, other
sizes, greedy generation through generate_step."""
import math

import numpy as np
import pytest
import torch

import negosun_oracle as O

pytestmark = pytest.mark.gpu

F32_TOL = 2e-4        # float32 model against the float64 oracle (centred rms over the vocabulary, relative)
BF16_TOL = 6e-2       # bfloat16 matrix products
I32 = dict(dtype=torch.int32, device="cuda")


def build(cfg, seed=0, dtype=torch.float32, weights=None, gain=1.0):
    from mlx_parallm_b200.utils import _get_classes
    Model, Args = _get_classes(cfg)
    w = O.random_weights(cfg, seed, gain=gain) if weights is None else weights
    return Model(Args.from_dict(cfg)).load_weights(w, device="cuda", dtype=dtype), w


def toks(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def residuals(cfg, w, t):
    res = []
    logits = O.forward(cfg, w, t, tap=lambda run, x: res.append(x.clone()))
    return logits, res


CONFIGS = {
    # every branch: layers with and without value mixing, temperature, feed-forward, shared expert and expert groups; grouped heads
    "mixed": lambda: O.make_config([
        O.layer(4, 2, 8, 12, 0.35, v_mix=False, q_temp=(0.4, 6), mlp=O.moe_mlp(6, 2, 16, (3, 2), shared=20)),
        O.layer(6, 2, 12, 8, 0.3, q_temp=(0.8, 5), mlp=O.moe_mlp(8, 3, 12, (4, 2))),
        O.layer(4, 1, 8, 16, 0.4, q_temp=None, mlp=O.moe_mlp(4, 2, 12, shared=8)),
        O.layer(2, 2, 16, 4, 0.25, v_mix=False),
        O.layer(2, 2, 8, 8, 0.35, q_temp=(0.3, 1), mlp=O.moe_mlp(9, 4, 8, (3, 3), shared=16)),
    ]),
    # sizes off the fast paths (odd width, heads, values), every expert chosen, one group kept, no cap on the logits
    "odd": lambda: O.make_config([
        O.layer(3, 1, 5, 7, 0.4, q_temp=(0.5, 3), mlp=O.moe_mlp(4, 4, 13, shared=5)),
        O.layer(7, 7, 3, 1, 0.45, q_temp=(1.1, 11), mlp=O.moe_mlp(10, 3, 9, (2, 1), shared=7)),
        O.layer(5, 1, 6, 7, 0.3, mlp=O.moe_mlp(7, 2, 9, (7, 5))),
    ], vocab=31, width=27, eps=1e-3, mult=1.0, softcap=None),
    # heads of the tile kernels' sizes, more than 16 query heads on one key head
    "wide": lambda: O.make_config([
        O.layer(4, 2, 64, 32, 0.12, q_temp=(0.2, 64), mlp=O.moe_mlp(4, 1, 24, (2, 1), shared=32)),
        O.layer(20, 1, 32, 64, 0.17, q_temp=(0.2, 100), mlp=O.moe_mlp(8, 2, 16, (4, 3), shared=24)),
        O.layer(2, 2, 96, 32, 0.1, mlp=O.moe_mlp(3, 2, 40)),
    ], vocab=130, width=64, mult=0.4, softcap=5.0),
    # one head, one expert, nothing optional
    "plain": lambda: O.make_config([O.layer(1, 1, 8, 8, 0.35, v_mix=False, q_temp=None, mlp=O.moe_mlp(1, 1, 24)),
                                    O.layer(1, 1, 8, 8, 0.3, v_mix=False, q_temp=None)], vocab=50, width=32, mult=0.9, softcap=None),
}


@pytest.fixture(scope="module")
def models():
    out = {}
    for name, mk in CONFIGS.items():
        cfg = mk()
        m, w = build(cfg, seed=len(name))
        out[name] = (cfg, m, w)
    return out


# ---- the residual step ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("W,M", [(32, 5), (27, 9), (512, 4), (1024, 3), (2048, 5), (4096, 2), (4096, 300), (6000, 3), (10240, 2), (200, 700), (2050, 3)])
def test_residual_step_with_channel_scales_and_two_norms(W, M):
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(W + M)
    h0, y1, y2 = (torch.randn(M, W, generator=g) for _ in range(3))
    s1, s2, w1, w2 = (1.0 + 0.3 * torch.randn(W, generator=g) for _ in range(4))
    eps, d = 1e-3, lambda t: t.double()
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2), (torch.float16, 2e-3)):
        for a, b in ((y1, y2), (y1, None), (None, y2), (None, None)):
            h = h0.cuda()
            x, x2 = (torch.full((M, W), 9.0, dtype=dt, device="cuda") for _ in range(2))
            raw = torch.full((M, 2 * W), 7.0, dtype=dt, device="cuda")
            ops.residual_add_norm(h, eps, dt, y1=None if a is None else a.cuda(), c1=0.3, y2=None if b is None else b.cuda(), c2=-0.7,
                                  s1=s1.cuda(), s2=s2.cuda(), w_next=w1.cuda(), x_out=x, w_next2=w2.cuda(), x_out2=x2, raw_out=raw[:, :W])
            want = d(h0) + (0 if a is None else 0.3 * d(s1) * d(a)) + (0 if b is None else -0.7 * d(s2) * d(b))
            assert (d(h.cpu()) - want).abs().max() < 1e-5 * max(1.0, float(want.abs().max()))
            assert torch.equal(raw[:, :W], h.to(dt)) and float((raw[:, W:].float() - 7.0).abs().max()) == 0.0
            for got, w in ((x, w1), (x2, w2)):
                ref = O.norm(want, d(w), eps)
                assert (d(got.cpu()) - ref).abs().max() < tol * max(1.0, float(ref.abs().max()))
        h = h0.cuda()
        ops.residual_add_norm(h, eps, dt, y1=y1.cuda(), s1=s1.cuda(), w_next2=w2.cuda(), x_out2=x2)      # one scaled branch, only a second reader
        want = d(h0) + d(s1) * d(y1)
        assert (d(h.cpu()) - want).abs().max() < 1e-5 * max(1.0, float(want.abs().max()))
        assert (d(x2.cpu()) - O.norm(want, d(w2), eps)).abs().max() < tol * 6.0


# ---- feed-forward ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,M,groups", [(6, 2, 9, (3, 2)), (12, 1, 40, (4, 1)), (5, 5, 3, (1, 1)), (40, 7, 33, (8, 3)), (1, 1, 4, (1, 1)),
                                            (130, 3, 20, (13, 2)), (16, 4, 50, (16, 5)), (64, 8, 21, (2, 1)), (15, 4, 30, (5, 5))])
def test_routing_inside_the_best_groups(E, top, M, groups):
    """Experts of the groups with the largest single score, weights over the chosen scores' sum; far logits do not break the choice,
    and a group of many good experts loses against one with a single better one."""
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(E * 10 + top)
    logits = torch.randn(M, E, generator=g) * 2.0
    logits[0] *= 30.0
    count, keep = groups
    if count > 1 and keep < count and E // count > 1:
        per = E // count
        logits[1] = torch.linspace(0.0, 0.01, E)
        logits[1, ::per] += torch.arange(1, count + 1).float()                 # every group's best expert decides
        logits[1, :per] = float(count - keep) + 0.5 + torch.linspace(0.0, 0.02, per)       # the first group: all good, none best: its sum would win
    ids = torch.zeros(M, top, **I32)
    wts = torch.zeros(M, top, device="cuda")
    seg, slot_of, token_of = torch.zeros(E + 1, **I32), torch.zeros(M, top, **I32), torch.zeros(M, top, **I32)
    ops.moe_route_scores(logits.cuda(), ids, wts, seg, slot_of, token_of, top, softmax=True, groups=count, keep=keep, renorm=True)
    # the float64 softmax of the scaled row keeps the scores apart, so the oracle's choice is the definition's
    want_ids, want_w = O.route(logits.double(), top, {"count": count, "keep": keep})
    assert ids.cpu().tolist()[1:] == want_ids.tolist()[1:]
    assert (wts.cpu().double() - want_w)[1:].abs().max() < 1e-6
    assert ids.cpu()[0, 0] == want_ids[0, 0] and abs(float(wts[0].sum()) - 1.0) < 1e-6 and (wts.cpu().double() - want_w)[0].abs().max() < 1e-5
    counts = torch.bincount(ids.cpu().flatten().long(), minlength=E)
    assert seg.cpu().tolist() == [0] + torch.cumsum(counts, 0).tolist()
    # sigmoid scores by the same rule
    ops.moe_route_scores(logits.cuda(), ids, wts, seg, slot_of, token_of, top, groups=count, keep=keep, renorm=True)
    s = torch.sigmoid(logits[1:].double())
    w, i = torch.topk(s.masked_fill(~O.open_experts(s, count, keep), -1.0), top, dim=-1)
    assert ids.cpu()[1:].tolist() == i.tolist() and (wts.cpu()[1:].double() - w / w.sum(-1, keepdim=True)).abs().max() < 1e-6


@pytest.mark.parametrize("E,N,K,tokens,top", [(16, 256, 128, 32, 2), (16, 2048, 192, 5, 1), (40, 128, 64, 64, 3), (8, 1000, 72, 17, 2), (160, 136, 256, 33, 4),
                                              (3, 6400, 64, 40, 1), (300, 96, 128, 64, 6), (4, 64, 48, 9, 2)])
def test_grouped_products_of_few_rows(E, N, K, tokens, top):
    """The experts' products of a decode step, with and without the gated unit: groups of unequal sizes, some empty, one with every
    token; rows beyond the groups' are not written."""
    from mlx_parallm_b200 import _lib, ops
    g = torch.Generator().manual_seed(E + N)
    pick = torch.randint(0, E, (tokens * top,), generator=g)
    pick[:tokens] = E // 2
    pick[tokens:] = torch.where(pick[tokens:] == E // 2, (E // 2 + 1) % E, pick[tokens:])
    cnt = torch.bincount(pick, minlength=E)
    cnt[cnt > tokens] = tokens
    seg = torch.cat([torch.zeros(1, dtype=torch.long), torch.cumsum(cnt, 0)])
    total = tokens * top
    for dt, tol in ((torch.bfloat16, 1e-2), (torch.float16, 2e-3), (torch.float32, 1e-5)):
        x = torch.randn(total, K, generator=g).to(dt)
        w = (torch.randn(E, N, K, generator=g) / math.sqrt(K)).to(dt)
        for epi in (_lib.GEMM_STORE_F32, _lib.GEMM_GLU_SILU):
            n_out = N // 2 if epi == _lib.GEMM_GLU_SILU else N
            out = torch.full((total, n_out), 5.0, dtype=torch.float32 if epi == _lib.GEMM_STORE_F32 else dt, device="cuda")
            ops.gemm_grouped(x.cuda(), w.cuda(), seg.to(torch.int32).cuda(), tokens, epi, out=out)
            got = out.double().cpu()
            for e in range(E):
                lo, hi = int(seg[e]), int(seg[e + 1])
                z = x[lo:hi].double() @ w[e].double().T
                want = z if epi == _lib.GEMM_STORE_F32 else O.silu(z[:, 0::2]) * z[:, 1::2]
                t = 1e-5 if epi == _lib.GEMM_STORE_F32 else tol
                assert hi == lo or (got[lo:hi] - want).abs().max() < t * max(1.0, float(want.abs().max())), (e, epi)
            assert int(seg[-1]) == total or float((got[int(seg[-1]):] - 5.0).abs().max()) == 0.0
    assert _lib.lib().b200p_gemm_tc_fault() == 0


@pytest.mark.parametrize("M,W,top,shared", [(5, 27, 2, True), (33, 64, 4, False), (300, 1024, 3, True), (4, 4100, 1, True)])
def test_expert_outputs_combined(M, W, top, shared):
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(W)
    ye, ysh = torch.randn(M * top, W, generator=g), torch.randn(M, W, generator=g)
    slot = torch.randperm(M * top, generator=g).view(M, top)
    wts = torch.rand(M, top, generator=g)
    y = torch.zeros(M, W, device="cuda")
    ops.moe_combine(ye.cuda(), slot.to(torch.int32).cuda(), wts.cuda(), ysh.cuda() if shared else None, y, top)
    want = (wts.double().unsqueeze(-1) * ye.double()[slot]).sum(1) + (ysh.double() if shared else 0.0)
    assert (y.double().cpu() - want).abs().max() < 1e-5


# ---- the head ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("M,N,K", [(1, 31, 27), (3, 130, 64), (9, 1000, 128), (32, 4000, 256), (64, 320, 96), (200, 257, 64), (700, 512, 128)])
def test_capped_logits_on_every_product_path(M, N, K):
    from mlx_parallm_b200 import _lib, ops
    g = torch.Generator().manual_seed(M + N)
    for dt in (torch.float32, torch.bfloat16, torch.float16):
        x = (torch.randn(M, K, generator=g) * torch.logspace(-3, 1.5, M).unsqueeze(1)).to(dt)
        w = (torch.randn(N, K, generator=g) / math.sqrt(K) * 3).to(dt)
        for cap in (0.7, 30.0):
            out = ops.gemm(x.cuda(), w.cuda(), _lib.GEMM_CAP_F32, act=(cap, 0.0))
            assert out.dtype == torch.float32
            z = x.double() @ w.double().T
            mag = x.double().abs() @ w.double().abs().T
            assert ((out.double().cpu() - O.cap(z, cap)).abs() <= 2e-6 * mag + 1e-6 * cap).all() and float(out.abs().max()) <= cap
    assert _lib.lib().b200p_gemm_tc_fault() == 0


# ---- attention --------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,G,d,dv,temp,blend,keep", [(3, 1, 6, 5, (0.5, 7), True, False), (4, 2, 16, 8, None, False, True), (4, 4, 64, 64, (1.5, 1), True, True),
                                                      (6, 1, 96, 48, (0.1, 600), False, False), (5, 5, 12, 4, (0.25, 5000), True, False)])
def test_attention_preparation(H, G, d, dv, temp, blend, keep):
    """Biases, whole-row norms, the temperature just before and at a step of its logarithm, values blended and kept, the places written."""
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(H + d)
    pos = [0, 1, 5, 6, 7, 599, 598, 4999, 5000]
    M, n = len(pos), H * d + G * d + G * dv
    proj = torch.randn(M, (n + 7) // 8 * 8, generator=g)
    bias, wq, wk = torch.randn(n, generator=g), torch.rand(H * d, generator=g) + 0.5, torch.rand(G * d, generator=g) + 0.5
    first = torch.randn(M, G * dv, generator=g)
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        q, kept = torch.zeros(M, H * d, device="cuda"), torch.zeros(M, G * dv, device="cuda")
        kc, vc = torch.full((2, G, 5003, d), 5.0, dtype=dt, device="cuda"), torch.full((2, G, 5003, dv), 5.0, dtype=dt, device="cuda")
        ops.row_attn_prep(proj.cuda(), 0, H * d, (H + G) * d, bias.cuda(), wq.cuda(), wk.cuda(), 1e-3, None, 0, 1.0, False, 0.3, q, kc, vc,
                          torch.ones(M, **I32), torch.tensor(pos, **I32), H, G, d, dv, *(temp or ()), v_first=first.cuda() if blend else None,
                          v_lambda=0.35, v_keep=kept if keep else None)
        p = proj[:, :n].double() + bias.double()
        qd, kd, vd = p[:, :H * d], p[:, H * d:(H + G) * d], p[:, (H + G) * d:]
        t = O.query_temperature(5001, {"coef": temp[0], "every": temp[1]} if temp else None)[pos]
        wantq = O.norm(qd, wq.double(), 1e-3) * t.unsqueeze(1) * 0.3
        wantk, wantv = O.norm(kd, wk.double(), 1e-3), O.blend_values(vd, first.double() if blend else None, 0.35)
        assert (q.double().cpu() - wantq).abs().max() < 1e-5 * max(1.0, float(wantq.abs().max()))
        assert (kc[1][:, pos].double().cpu().transpose(0, 1).reshape(M, -1) - wantk).abs().max() < tol * float(wantk.abs().max())
        assert (vc[1][:, pos].double().cpu().transpose(0, 1).reshape(M, -1) - wantv).abs().max() < tol * float(wantv.abs().max())
        assert float((kc[0].float() - 5.0).abs().max()) == 0.0 and float((vc[1][:, 8:598].float() - 5.0).abs().max()) == 0.0
        assert (kept.double().cpu() - (wantv if keep else 0.0)).abs().max() < 1e-5 * max(1.0, float(wantv.abs().max()))


def attn_case(T, H, G, d, dv, hot, dtype, start=0, decode=False, seed=0, workspace=True):
    """Attention over T cached positions of row 1; tokens start .. T-1 are the queries.  One query / key pair stands out, so that a
    key that is wrongly masked, skipped or misplaced shows.  Rows and positions behind the sequence hold large values."""
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(seed + T + H)
    q, k, v = torch.randn(T, H, d, generator=g) * 0.3, torch.randn(T, G, d, generator=g) * 0.3, torch.randn(T, G, dv, generator=g)
    if hot is not None:
        u = torch.randn(d, generator=g)
        u = u / u.norm()
        q[hot[0]] += 10.0 * u
        k[hot[1]] += 3.0 * u
    q, k, v = (x.to(dtype).float() for x in (q, k, v))
    cap = T + 70
    kc, vc = torch.full((3, G, cap, d), 3.0), torch.full((3, G, cap, dv), 50.0)
    kc[1, :, :T], vc[1, :, :T] = k.transpose(0, 1), v.transpose(0, 1)
    kc, vc = kc.to(dtype).cuda(), vc.to(dtype).cuda()
    qs = q[start:].reshape(T - start, H * d).contiguous().cuda()
    n = T - start
    out = torch.zeros(n, H * dv, dtype=dtype, device="cuda")
    ws = torch.zeros(ops.sink_attn_workspace_floats(1, H, dv), device="cuda") if workspace else None
    for lo, hi in ([(i, i + 1) for i in range(n)] if decode else [(0, n)]):
        ops.sink_attn(qs[lo:hi], kc, vc, torch.ones(hi - lo, **I32), torch.arange(start + lo, start + hi, **I32), None, 0.0, out[lo:hi], H, G, d, dv,
                      1.0, cu=torch.tensor([0, hi - lo], **I32), rows=torch.tensor([1], **I32), nb=1, max_n=hi - lo, workspace=ws)
    want = O.causal_attention(q.double(), k.double(), v.double(), 1.0)[start:]
    if hot is not None and hot[1] <= hot[0]:           # the standing-out key really decides
        assert (want[hot[0] - start] - v.double()[hot[1]].repeat_interleave(H // G, 0)).abs().max() < 0.05
    return (out.double().cpu().view(n, H, dv) - want).abs().max()


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 96, 32), (8, 1, 96, 96), (4, 4, 32, 32), (6, 2, 32, 128), (4, 1, 64, 96), (2, 2, 128, 32), (4, 2, 96, 64),
                                      (4, 2, 64, 64), (4, 1, 128, 128), (3, 3, 96, 128), (2, 1, 64, 32), (2, 1, 32, 64), (2, 1, 128, 96), (3, 1, 32, 96),
                                      (5, 1, 7, 9), (2, 2, 80, 48)])
def test_attention_sizes_far_keys_and_tile_borders(H, G, d, dv):
    for T, start, hot in ((200, 0, (199, 0)), (130, 0, (129, 64)), (130, 0, (127, 63)), (130, 0, (64, 64)), (130, 0, (64, 65)), (65, 0, (64, 0)),
                          (64, 60, (63, 1)), (300, 255, (299, 128)), (5, 0, (4, 0)), (2, 0, (1, 0)), (3, 1, (2, 2))):
        for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2), (torch.float16, 5e-3)):
            assert attn_case(T, H, G, d, dv, hot, dtype, start) < tol, (T, start, hot, dtype)


@pytest.mark.parametrize("H,G,d,dv", [(9, 1, 96, 32), (16, 1, 32, 32), (17, 1, 64, 64), (40, 1, 96, 64), (48, 2, 64, 32), (36, 2, 128, 128), (32, 1, 128, 32),
                                      (6, 3, 32, 96), (20, 1, 10, 6)])
def test_decode_attention_of_many_heads_per_key_head(H, G, d, dv):
    """One token against split keys, blocks of 16 heads: keys at the first and last position and at tile borders."""
    for T, hot in ((1, (0, 0)), (2, (1, 0)), (64, (63, 0)), (65, (64, 64)), (66, (65, 64)), (129, (128, 63)), (1100, (1099, 0)), (1100, (1099, 1023)),
                   (1100, (1099, 1099))):
        for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 3e-2)):
            assert attn_case(T, H, G, d, dv, hot, dtype, T - 1, decode=True) < tol, (T, hot, dtype)
    assert attn_case(70, H, G, d, dv, (69, 3), torch.bfloat16, 60, decode=True, workspace=False) < 3e-2


def single(cfg, w, T, seed, dtype=torch.float32, cuts=None):
    m, _ = build(cfg, dtype=dtype, weights=w)
    t = toks(cfg, T, seed)
    _, res = residuals(cfg, w, t)
    got = []
    m.residual_tap = lambda layer, kind, h: got.append((layer, h.clone()))
    cache = m.make_cache(1)
    lo = 0
    for n in (cuts or [T]):
        m.forward_ragged([t[lo:lo + n]], cache)
        lo += n
    last = len(cfg["layers"]) - 1
    return torch.cat([h for i, h in got if i == last]).double().cpu(), res[last]


@pytest.mark.parametrize("H,G,dk,dv,temp", [(4, 2, 8, 12, (0.5, 5)), (3, 1, 5, 7, None), (2, 2, 64, 64, (1.0, 9)), (6, 3, 96, 32, (0.2, 1)), (20, 5, 8, 8, (0.5, 7)),
                                            (34, 1, 32, 32, (0.3, 20))])
def test_layers_alone(H, G, dk, dv, temp):
    """Attention by itself, and three layers whose values are blended with the first one's."""
    for layers in ([O.layer(H, G, dk, dv, 1.5 / math.sqrt(dk), v_mix=False, q_temp=temp)],
                   [O.layer(H, G, dk, dv, 1.5 / math.sqrt(dk), v_mix=i != 1, q_temp=temp) for i in range(4)]):
        cfg = O.make_config(layers, width=32)
        w = O.random_weights(cfg, H + dk)
        for dtype, tol in ((torch.float32, 2e-4), (torch.bfloat16, 6e-2)):
            for cuts in (None, [9, 1, 1, 2, 27]):
                got, want = single(cfg, w, 40, 3, dtype=dtype, cuts=cuts)
                assert (got - want).abs().max() < tol * max(1.0, float(want.abs().max()))


# ---- whole models -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_logits_and_residuals_match_the_oracle(models, name):
    cfg, m, w = models[name]
    t = toks(cfg, 45, 1)
    want, res = residuals(cfg, w, t)
    got_res = []
    m.residual_tap = lambda layer, kind, h: got_res.append((layer, h.clone()))
    try:
        got = m.forward_ragged([t], m.make_cache(1), want=[list(range(len(t)))])
    finally:
        m.residual_tap = None
    assert [i for i, _ in got_res] == list(range(len(cfg["layers"])))
    for k, r in enumerate(res):
        assert (got_res[k][1].double().cpu() - r).abs().max() < 2e-4 * max(1.0, float(r.abs().max())), f"residual after layer {k}"
    assert O.logits_error(got, want) < F32_TOL
    assert cfg["logit_softcap"] is None or float(got.abs().max()) <= cfg["logit_softcap"]


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float16])
def test_16_bit_models(name, dtype):
    cfg = CONFIGS[name]()
    m, w = build(cfg, seed=3, dtype=dtype, gain=0.7)
    t = toks(cfg, 60, 2)
    got = m.forward_ragged([t], m.make_cache(1), want=[list(range(len(t)))])
    want = O.forward(cfg, w, t)
    per_pos = sorted(O.logits_error(got[i:i + 1], want[i:i + 1]) for i in range(len(t)))       # rounding flips an expert now and then
    assert per_pos[len(t) // 2] < BF16_TOL and per_pos[-1] < 1.0, per_pos[-3:]


def test_bfloat16_model_on_the_tensor_core_paths():
    """Sizes the tile attention kernels and the tcgen05 grouped products take: a prompt, a ragged batch and decode steps through the
    captured step (two branches side by side) in bfloat16 against the oracle; positions compared by their typical error."""
    from mlx_parallm_b200 import utils
    cfg = O.make_config([
        O.layer(4, 2, 64, 64, 0.125, q_temp=(0.3, 50), mlp=O.moe_mlp(8, 2, 256, (4, 2), shared=128)),
        O.layer(32, 1, 32, 128, 0.17, mlp=O.moe_mlp(4, 1, 1024, (2, 1))),
        O.layer(4, 4, 96, 32, 0.1, q_temp=(0.2, 128), mlp=O.moe_mlp(6, 3, 128, (3, 2), shared=64)),
    ], vocab=200, width=128)
    m, w = build(cfg, seed=7, dtype=torch.bfloat16, gain=0.8)
    t = toks(cfg, 330, 3)
    want = O.forward(cfg, w, t)
    got = m.forward_ragged([t[:300]], m.make_cache(1), want=[list(range(300))])
    per_pos = sorted(O.logits_error(got[i:i + 1], want[i:i + 1]) for i in range(300))
    assert per_pos[150] < BF16_TOL and per_pos[-1] < 1.0, per_pos[-3:]
    lens = [300, 70, 5, 1, 2, 33, 64, 128, 200, 260, 11, 12]
    cache = utils._kv_pool.get_for(m, len(lens))
    rows = list(range(len(lens)))[::-1]
    first = m.forward_ragged([t[:n] for n in lens], cache, rows=rows)
    errs = [O.logits_error(first[i:i + 1], want[n - 1:n]) for i, n in enumerate(lens)]
    st = utils._decode_step_for(m, cache, len(lens), False)
    st.set_rows(rows)
    for k in range(30):
        st.tok.copy_(torch.tensor([t[n + k] for n in lens], dtype=torch.int32))
        st.run()
        errs += [O.logits_error(st.logits[i:i + 1], want[n + k:n + k + 1]) for i, n in enumerate(lens)]
    errs.sort()
    assert errs[len(errs) // 2] < BF16_TOL and errs[-1] < 1.0, errs[-3:]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 0.0), (torch.bfloat16, 2e-2)])
def test_branches_side_by_side_equal_one_after_the_other(dtype, tol):
    from mlx_parallm_b200 import utils
    cfg = CONFIGS["wide"]()
    m, w = build(cfg, seed=5, dtype=dtype)
    t = toks(cfg, 40, 6)
    out = []
    for overlap in (True, False):
        m.overlap_branches = overlap
        cache = m.make_cache(2)
        m.forward_ragged([t[:20], t[:7]], cache)
        st = utils.DecodeSession(m, cache, 2, greedy=False)
        rows = []
        for k in range(12):
            st.tok.copy_(torch.tensor([t[20 + k], t[7 + k]], dtype=torch.int32))
            st.run()
            rows.append(st.logits.clone())
        out.append(torch.cat(rows))
    assert O.logits_error(out[0], out[1]) <= tol


@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_and_single_tokens_equal_one_pass(models, name):
    """A prompt cut into portions of 1, 2, 3, ... tokens, and fed token by token, gives the logits of one pass."""
    cfg, m, w = models[name]
    t = toks(cfg, 50, 4)
    want = O.forward(cfg, w, t)
    for cuts in ([50], [1, 2, 3, 5, 8, 13, 18], [2] * 25, [1] * 50, [47, 1, 2], [49, 1], [33, 17], [3, 1, 1, 45]):
        cache = m.make_cache(3)
        got, lo = [], 0
        for n in cuts:
            got.append(m.forward_ragged([t[lo:lo + n]], cache, rows=[2], want=[list(range(n))]))
            lo += n
        assert O.logits_error(torch.cat(got), want) < F32_TOL, cuts


@pytest.mark.parametrize("name", ["mixed", "wide", "odd"])
def test_decode_step_graph_against_prompt(models, name):
    """Most of a prompt in one pass, the rest through the engine's captured decode step (the generation path)."""
    from mlx_parallm_b200 import utils
    cfg, m, w = models[name]
    t = toks(cfg, 100, 5)
    want = O.forward(cfg, w, t)
    cache = utils._kv_pool.get_for(m, 1)
    got = [m.forward_ragged([t[:30]], cache, want=[[29]])]
    st = utils._decode_step_for(m, cache, 1, False)
    for tok in t[30:]:
        st.tok.copy_(torch.tensor([tok], dtype=torch.int32))
        st.run()
        got.append(st.logits.clone())
    assert O.logits_error(torch.cat(got), want[29:]) < F32_TOL
    assert cache[-1].offsets == [100]


def test_ragged_batch_equals_each_alone_and_rows_end_early(models):
    """Four prompts of 1, 2, 17 and 40 tokens in one pass, then decoded together while the short ones end: equal to each request
    alone in a cache of its own, and right against the oracle."""
    from mlx_parallm_b200 import utils
    cfg, m, w = models["mixed"]
    lens, extra = [1, 2, 17, 40], [0, 3, 12, 12]
    seqs = [toks(cfg, n + e, 10 + n) for n, e in zip(lens, extra)]
    cache = utils._kv_pool.get_for(m, 4)
    rows = [2, 0, 3, 1]
    first = m.forward_ragged([s[:n] for s, n in zip(seqs, lens)], cache, rows=rows, want=[list(range(n)) for n in lens])
    together = {i: [] for i in range(4)}
    o = 0
    for i, n in enumerate(lens):
        together[i].append(first[o:o + n])
        o += n
    m.release_rows(cache, [rows[0]])
    for k in range(12):
        live = [i for i in range(1, 4) if k < extra[i]]
        st = utils._decode_step_for(m, cache, len(live), False)
        st.set_rows([rows[i] for i in live])
        st.tok.copy_(torch.tensor([seqs[i][lens[i] + k] for i in live], dtype=torch.int32))
        st.run()
        for j, i in enumerate(live):
            together[i].append(st.logits[j:j + 1].clone())
        if k + 1 == extra[1]:
            m.release_rows(cache, [rows[1]])
    for i in range(4):
        got = torch.cat(together[i])
        assert O.logits_error(got, O.forward(cfg, w, seqs[i])) < F32_TOL
        alone_cache = m.make_cache(1)
        alone = [m.forward_ragged([seqs[i][:lens[i]]], alone_cache, want=[list(range(lens[i]))])]
        for tok in seqs[i][lens[i]:]:
            alone.append(m.forward_ragged([[tok]], alone_cache))
        assert torch.equal(torch.cat(alone), got), f"request {i} depends on its batch"


def test_bfloat16_ragged_batch_of_unequal_requests():
    """The tile kernels over a ragged batch: every request's positions as the oracle says, up to 16-bit rounding."""
    cfg = O.make_config([O.layer(6, 2, 64, 64, 0.125), O.layer(8, 1, 96, 128, 0.1, q_temp=(0.3, 40)),
                         O.layer(20, 2, 32, 64, 0.17)], vocab=90, width=64)
    m, w = build(cfg, seed=2, dtype=torch.bfloat16, gain=0.8)
    seqs = [toks(cfg, n, n) for n in (3, 130, 16, 1, 65)]
    got = m.forward_ragged(seqs, m.make_cache(5), want=[list(range(len(s))) for s in seqs])
    o = 0
    for s in seqs:
        want = O.forward(cfg, w, s)
        errs = sorted(O.logits_error(got[o + i:o + i + 1], want[i:i + 1]) for i in range(len(s)))
        assert errs[-1] < BF16_TOL, (len(s), errs[-3:])
        o += len(s)


def test_rows_given_back_start_from_nothing(models):
    """A row that held a long sequence is released and takes a new one, alone and beside a row that goes on."""
    for name in ("mixed", "wide", "plain"):
        cfg, m, w = models[name]
        cache = m.make_cache(2)
        old, keep, new = toks(cfg, 60, 20), toks(cfg, 30, 21), toks(cfg, 25, 22)
        m.forward_ragged([old, keep[:20]], cache)
        m.release_rows(cache, [0])
        assert cache[0].offsets == [0, 20]
        got = m.forward_ragged([new[:3], keep[20:]], cache, want=[[0, 1, 2], list(range(10))])
        assert O.logits_error(got[:3], O.forward(cfg, w, new)[:3]) < F32_TOL
        assert O.logits_error(got[3:], O.forward(cfg, w, keep)[20:]) < F32_TOL
        rest = m.forward_ragged([new[3:]], cache, rows=[0], want=[list(range(22))])
        assert O.logits_error(rest, O.forward(cfg, w, new)[3:]) < F32_TOL
        m.release_rows(cache, [0])
        one = torch.cat([m.forward_ragged([[tok]], cache, rows=[0]) for tok in new[:6]])
        assert O.logits_error(one, O.forward(cfg, w, new[:6])) < F32_TOL


def test_first_tokens_and_short_sequences(models):
    for name in ("mixed", "odd", "plain"):
        cfg, m, w = models[name]
        seqs = [toks(cfg, n, 30 + n) for n in (1, 1, 2, 3, 4)]
        got = m.forward_ragged(seqs, m.make_cache(5), want=[list(range(len(s))) for s in seqs])
        want = torch.cat([O.forward(cfg, w, s) for s in seqs])
        assert O.logits_error(got, want) < F32_TOL


def test_far_keys_in_the_model_and_a_growing_cache():
    """A sharp softmax over 620 positions: answers at the end change clearly when the first token changes.  Fed in portions that end
    just before, at and just after the cache's growth at 256 and 512 positions, then token by token."""
    cfg = O.make_config([O.layer(2, 1, 16, 16, 2.0, q_temp=(1.0, 60)), O.layer(2, 2, 8, 8, 1.0)], vocab=40, width=32)
    w = O.random_weights(cfg, 12)
    m, _ = build(cfg, weights=w)
    t = toks(cfg, 620, 3)
    a = O.forward(cfg, w, t)
    u = next(x for x in range(40) if O.logits_error(O.forward(cfg, w, [x] + t[1:])[-10:], a[-10:]) > 5e-3)
    t = [u] + t[1:]
    want = O.forward(cfg, w, t)
    for cuts in ([255, 1, 1, 254, 1, 1, 97], [256, 256, 98], [257, 254, 2, 97], [610]):
        cache = m.make_cache(1)
        lo = 0
        for n in cuts:
            m.forward_ragged([t[lo:lo + n]], cache)
            lo += n
        got = torch.cat([m.forward_ragged([[tok]], cache) for tok in t[lo:]])
        assert lo == 610 and O.logits_error(got, want[lo:]) < F32_TOL, cuts


def test_query_temperature_shows_in_the_model():
    """With the temperature left out, or its blocks one token off, the answers differ by far more than the tolerance."""
    cfg = O.make_config([O.layer(4, 2, 16, 16, 0.5, q_temp=(1.5, 10))], vocab=40, width=32)
    w = O.random_weights(cfg, 4)
    m, _ = build(cfg, weights=w)
    t = toks(cfg, 45, 7)
    want = O.forward(cfg, w, t)
    assert O.logits_error(m.forward_ragged([t], m.make_cache(1), want=[list(range(45))]), want) < F32_TOL
    for other in (None, {"coef": 1.5, "every": 11}):
        c2 = O.make_config([dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], q_temp=other))], vocab=40, width=32)
        assert O.logits_error(O.forward(c2, w, t), want) > 20 * F32_TOL


def test_long_decoding(models):
    from mlx_parallm_b200 import utils
    cfg, m, w = models["odd"]
    t = toks(cfg, 330, 8)
    want = O.forward(cfg, w, t)
    cache = utils._kv_pool.get_for(m, 1)
    m.forward_ragged([t[:5]], cache)
    st = utils._decode_step_for(m, cache, 1, False)
    got = []
    for tok in t[5:]:
        st.tok.copy_(torch.tensor([tok], dtype=torch.int32))
        st.run()
        got.append(st.logits.clone())
    assert O.logits_error(torch.cat(got), want[5:]) < F32_TOL


def test_greedy_generation_through_generate_step(models):
    """The engine's own entry point: left-padded prompts with their lengths, prefill, then the captured decode step feeding its own
    argmax back.  Compared with greedy decoding of the oracle, request by request."""
    from mlx_parallm_b200 import utils
    cfg, m, w = models["mixed"]
    prompts = [toks(cfg, n, 40 + n) for n in (3, 9, 6)]
    L = max(len(p) for p in prompts)
    padded = torch.tensor([[0] * (L - len(p)) + p for p in prompts])
    n_new = 8
    gen = utils.generate_step(padded, m, prompt_lengths=[len(p) for p in prompts])
    got = torch.cat([y for _, (y, _) in zip(range(n_new), gen)], 1).cpu().tolist()
    for p, g in zip(prompts, got):
        seq = list(p)
        for tok in g:
            lg = O.forward(cfg, w, seq)[-1]
            best = int(lg.argmax())
            assert tok == best or float(lg[best] - lg[tok]) < 1e-3 * float(lg.abs().max())
            seq.append(tok)


def test_batch_generate_front_end(models):
    from fake_tokenizer import FakeTokenizer
    from mlx_parallm_b200 import utils
    from mlx_parallm_b200.tokenizer_utils import TokenizerWrapper
    cfg, m, w = models["mixed"]
    tok = TokenizerWrapper(FakeTokenizer(vocab_size=cfg["vocab"]))
    out = utils.batch_generate(m, tok, ["w5 w6", "w5 w6 w7 w8 w9 w10 w11"], max_tokens=5, format_prompts=False)
    alone = utils.batch_generate(m, tok, ["w5 w6"], max_tokens=5, format_prompts=False)
    assert len(out) == 2 and out[0] == alone[0]


def test_checkpoint_on_disk_and_trace_runner(tmp_path, models):
    """config.json + model.safetensors through load_model (the registry picks the class by the architecture's name), then the
    command-line trace runner on the same folder: prompt, decode steps and a request that ends early, against the oracle."""
    import json
    import os
    import subprocess
    import sys
    from safetensors.torch import save_file
    cfg, _, w = models["odd"]
    d = tmp_path / "model"
    d.mkdir()
    (d / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, str(d / "model.safetensors"))
    wb = {k: v.to(torch.bfloat16) for k, v in w.items()}
    a, b = toks(cfg, 12, 1), toks(cfg, 5, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:9], "want": [0, 8]}, {"id": "b", "tokens": b[:4], "want": [3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[9:10], "want": [0]}, {"id": "b", "tokens": b[4:5], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[10:11], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[11:12], "want": [0]}], "end": ["a"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(d), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                       timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.split("\n") if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wbb = O.forward(cfg, wb, a), O.forward(cfg, wb, b)
    V = cfg["vocab"]
    s0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(3, V))
    assert O.logits_error(s0, torch.stack([wa[0], wa[8], wbb[3]])) < F32_TOL
    s1 = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(1, V))
    assert O.logits_error(s1, wa[9:10]) < F32_TOL
    assert not (out / "2.f32").exists()
    s3 = torch.from_numpy(np.fromfile(out / "3.f32", dtype="<f4").reshape(1, V))
    assert O.logits_error(s3, wa[11:12]) < F32_TOL

"""Seradra on the GPU against the slow float64 oracle (tests/seradra_oracle.py): each mechanism alone, prompts against
token-by-token decoding, portions, ragged batches, rows given back and used again, far keys and window edges in prompts and in
decoding, the rotation, the depth averages, other sizes, greedy generation through generate_step."""
import math

import numpy as np
import pytest
import torch

import seradra_oracle as O

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
    # every branch: both mixers, dense and routed feed-forwards and none, grouped key heads, rotation with and without stretching
    "mixed": lambda: O.make_config([
        O.attention_layer(6, 2, 8, 12, 0.35, 11, 4, base=100.0, scaling=(4.0, 24, 6.0, 0.5), mlp=O.dense_mlp(24)),
        O.latent_layer(4, 8, 4, 12, 12, 16, 0.3, 9, mlp=O.moe_mlp(8, 3, 16)),
        O.attention_layer(4, 4, 16, 8, 0.25, 7, 16),
        O.latent_layer(2, 16, 8, 8, 8, 24, 0.2, 17, mlp=O.dense_mlp(20)),
        O.attention_layer(2, 1, 8, 8, 0.4, 30, 6, mlp=O.moe_mlp(5, 1, 20)),
    ]),
    # sizes off the fast paths (odd width, heads, value sizes), one key head for three heads, two rotated dimensions, every expert
    # chosen, windows of one and two positions
    "odd": lambda: O.make_config([
        O.attention_layer(3, 1, 5, 7, 0.4, 1, 2, base=7.0, scaling=(2.0, 8, 4.0, 1.0), mlp=O.moe_mlp(4, 4, 13)),
        O.latent_layer(3, 5, 2, 7, 9, 11, 0.45, 2, base=7.0, mlp=O.dense_mlp(15)),
        O.attention_layer(5, 5, 6, 3, 0.3, 13, 6, mlp=O.moe_mlp(7, 2, 9)),
    ], vocab=31, width=27, eps=1e-3),
    # wider heads: sizes of the tile kernels, a window longer than any test prompt, a latent row that fills its padding exactly
    "wide": lambda: O.make_config([
        O.attention_layer(4, 2, 64, 64, 0.12, 4096, 32, base=1e5, scaling=(8.0, 64, 16.0, 1.0), mlp=O.moe_mlp(3, 1, 24)),
        O.latent_layer(8, 32, 32, 32, 48, 96, 0.12, 20, base=1e5, mlp=O.dense_mlp(40)),
        O.attention_layer(3, 3, 128, 64, 0.09, 25, 128, mlp=O.dense_mlp(48)),
        O.latent_layer(8, 16, 8, 16, 24, 40, 0.2, 4096, mlp=O.moe_mlp(4, 2, 16)),
    ], vocab=130, width=64),
    # one head, one expert, no rotation, no window on either mixer, no feed-forward on the last layer
    "plain": lambda: O.make_config([
        O.attention_layer(1, 1, 8, 8, 0.35, 0, 0, mlp=O.moe_mlp(1, 1, 24)),
        O.latent_layer(1, 8, 8, 8, 8, 8, 0.3, 0),
    ], vocab=50, width=32),
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
@pytest.mark.parametrize("W,M", [(32, 5), (27, 9), (1024, 3), (4096, 2), (4096, 600), (10240, 2), (200, 700)])
def test_residual_step_and_depth_average(W, M):
    """A norm on the embedding, a sublayer closed without and with an average, the last one without a slot; the stack holds the
    vectors before averaging."""
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(W + M)
    h0, y1, y2 = (torch.randn(M, W, generator=g) for _ in range(3))
    w0, w1, w2 = (1.0 + 0.3 * torch.randn(W, generator=g) for _ in range(3))
    a, b = torch.randn(2, generator=g), torch.randn(3, generator=g)
    eps = 1e-3
    d = lambda t: t.double()
    x0 = O.rms_unit(d(h0), eps) * d(w0)
    x1 = x0 + O.rms_unit(d(y1), eps) * d(w1)
    s1 = d(a)[0] * x0 + d(a)[1] * x1
    x2 = s1 + O.rms_unit(d(y2), eps) * d(w2)
    s2 = d(b)[0] * x0 + d(b)[1] * x1 + d(b)[2] * x2
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 1e-2)):
        h = h0.cuda()
        stack = torch.full((M, 2, W), 7.0, device="cuda")
        raw = torch.zeros(M, W, dtype=dt, device="cuda")
        ops.post_norm_step(h, w0.cuda(), eps, dt, stack=stack, slot=0, raw_out=raw)
        scale = max(1.0, float(x0.abs().max()))
        assert (d(h.cpu()) - x0).abs().max() < 1e-5 * scale and (d(raw.cpu()) - x0).abs().max() < tol * scale
        h1 = h.clone()
        ops.post_norm_step(h1, w1.cuda(), eps, dt, y=y1.cuda(), raw_out=raw)                       # no stack at all
        assert (d(h1.cpu()) - x1).abs().max() < 1e-5 * max(1.0, float(x1.abs().max()))
        assert float((stack[:, 1] - 7.0).abs().max()) == 0.0
        ops.post_norm_step(h, w1.cuda(), eps, dt, y=y1.cuda(), stack=stack, slot=1, avg=a.cuda(), raw_out=raw)
        assert (d(h.cpu()) - s1).abs().max() < 1e-5 * max(1.0, float(s1.abs().max()))
        assert (d(raw.cpu()) - s1).abs().max() < tol * max(1.0, float(s1.abs().max()))
        assert (d(stack.cpu()) - torch.stack([x0, x1], 1)).abs().max() < 1e-5 * max(1.0, float(x1.abs().max()))
        before = stack.clone()
        ops.post_norm_step(h, w2.cuda(), eps, dt, y=y2.cuda(), stack=stack, avg=b.cuda())
        assert (d(h.cpu()) - s2).abs().max() < 2e-5 * max(1.0, float(s2.abs().max())) and torch.equal(stack, before)


# ---- feed-forward ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("M,N,K", [(1, 24, 16), (5, 40, 27), (33, 96, 64), (300, 256, 128), (700, 512, 256)])
def test_two_parameter_activation(M, N, K):
    """Both sides of zero, large arguments, and arguments so small that e^z - 1 - z must not cancel, on every GEMM path."""
    from mlx_parallm_b200 import _lib, ops
    from mlx_parallm_b200.models._sequence import ActivatedFF
    g = torch.Generator().manual_seed(M + N)
    act = torch.tensor([0.7, -1.1])
    ff = ActivatedFF(K, N, "xielu")
    ff.set_xielu(act)
    for dt, tol in ((torch.float32, 2e-6), (torch.bfloat16, 1e-2), (torch.float16, 2e-3)):
        x = (torch.randn(M, K, generator=g) * torch.logspace(-4, 0.5, M).unsqueeze(1)).to(dt)
        w = (torch.randn(N, K, generator=g) / math.sqrt(K) * 2).to(dt)
        got = ops.gemm(x.cuda(), w.cuda(), _lib.GEMM_XIELU, act=ff.act_constants).double().cpu()
        z = x.double() @ w.double().T
        want = O.xielu(z, act.double())
        mag = x.double().abs() @ w.double().abs().T                  # what the sum's rounding is measured against
        slope = 0.5 + 2.5 * z.abs()                                  # the activation's slope
        sum_tol = 1e-6 * mag * slope                                 # fp32 accumulation
        store = (0.0 if dt == torch.float32 else tol) * want.abs()   # rounding of the result
        assert ((got - want).abs() <= sum_tol + store + 1e-6 * want.abs() + (0.0 if dt == torch.bfloat16 else 1e-9 if dt == torch.float32 else 1e-7)).all()


@pytest.mark.parametrize("E,top,M", [(6, 2, 9), (12, 1, 40), (5, 5, 3), (40, 7, 33), (1, 1, 4), (130, 3, 20)])
def test_routing_by_softmax_scores(E, top, M):
    """The chosen experts' weights are their softmax over ALL experts, not renormalised; far logits do not break the choice."""
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(E * 10 + top)
    logits = torch.randn(M, E, generator=g) * 2.0
    logits[0] *= 40.0                                                 # scores that underflow: picked by the logits all the same
    ids = torch.zeros(M, top, **I32)
    wts = torch.zeros(M, top, device="cuda")
    seg, slot_of, token_of = torch.zeros(E + 1, **I32), torch.zeros(M, top, **I32), torch.zeros(M, top, **I32)
    ops.moe_route_scores(logits.cuda(), ids, wts, seg, slot_of, token_of, top, softmax=True)
    _, want_ids = torch.topk(logits, top, dim=-1)
    want_w = torch.softmax(logits.double(), -1).gather(1, want_ids)
    assert ids.cpu().tolist() == want_ids.tolist()
    assert (wts.cpu().double() - want_w).abs().max() < 1e-6
    counts = torch.bincount(want_ids.flatten(), minlength=E)
    assert seg.cpu().tolist() == [0] + torch.cumsum(counts, 0).tolist()
    if top < E:
        assert float(wts[1:].sum(1).max()) < 1.0


# ---- mixers alone -----------------------------------------------------------------------------------------------------------
def mixer_alone(cfg, w, T, seed, dtype=torch.float32, cuts=None):
    """Residual stream after the single layer of cfg for T random tokens: framework (optionally fed in portions), oracle."""
    m, _ = build(cfg, dtype=dtype, weights=w)
    t = toks(cfg, T, seed)
    _, res = residuals(cfg, w, t)
    got = []
    m.residual_tap = lambda layer, kind, h: got.append(h.clone())
    cache = m.make_cache(1)
    lo = 0
    for n in (cuts or [T]):
        m.forward_ragged([t[lo:lo + n]], cache)
        lo += n
    m.residual_tap = None
    return torch.cat(got).double().cpu(), res[0]


@pytest.mark.parametrize("H,G,dk,dv,win,rot,scaling", [
    (4, 2, 8, 12, 5, 4, (4.0, 24, 6.0, 0.5)), (3, 1, 5, 7, 1, 2, None), (2, 2, 64, 64, 0, 64, (8.0, 64, 16.0, 1.0)), (6, 3, 48, 16, 9, 16, None),
    (1, 1, 128, 64, 20, 32, None), (8, 4, 64, 128, 4096, 8, (2.0, 8, 4.0, 1.0)), (20, 5, 8, 8, 13, 6, None), (40, 40, 4, 4, 11, 4, None)])
def test_mixed_score_attention_alone(H, G, dk, dv, win, rot, scaling):
    cfg = O.make_config([O.attention_layer(H, G, dk, dv, 1.5 / math.sqrt(dk), win, rot, base=50.0, scaling=scaling)], width=32)
    w = O.random_weights(cfg, H + dk)
    for cuts in (None, [9, 1, 1, 2, 27]):
        got, want = mixer_alone(cfg, w, 40, 3, cuts=cuts)
        assert (got - want).abs().max() < 2e-4 * max(1.0, float(want.abs().max()))
    for cuts in (None, [9, 1, 1, 2, 27]):
        got, want = mixer_alone(cfg, w, 40, 3, dtype=torch.bfloat16, cuts=cuts)
        assert (got - want).abs().max() < 6e-2 * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("H,dn,dr,dv,qr,kr,win", [(4, 8, 4, 12, 12, 16, 7), (3, 5, 2, 7, 9, 11, 1), (8, 32, 32, 32, 48, 96, 20),
                                                  (2, 64, 16, 64, 16, 48, 33), (1, 8, 8, 8, 8, 8, 0), (9, 8, 6, 8, 8, 600, 12)])
def test_windowed_latent_attention_alone(H, dn, dr, dv, qr, kr, win):
    cfg = O.make_config([O.latent_layer(H, dn, dr, dv, qr, kr, 1.2 / math.sqrt(dn + dr), win, base=50.0)], width=32)
    w = O.random_weights(cfg, H + kr)
    for dtype, tol in ((torch.float32, 2e-4), (torch.bfloat16, 6e-2)):
        for cuts in (None, [9, 1, 1, 2, 27]):
            got, want = mixer_alone(cfg, w, 40, 2, dtype=dtype, cuts=cuts)
            assert (got - want).abs().max() < tol * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("H,G,d,dv,n_rot,pairs,bias,normed", [(3, 1, 6, 5, 2, False, True, True), (4, 2, 16, 8, 8, False, True, True),
                                                              (4, 4, 64, 64, 16, False, False, True), (2, 2, 8, 8, 3, True, True, False),
                                                              (6, 2, 32, 16, 0, False, True, True), (2, 1, 24, 12, 4, False, True, False)])
def test_attention_preparation(H, G, d, dv, n_rot, pairs, bias, normed):
    """Biases, norms over whole rows, both rotation layouts, the magnitude, positions up to 5000, every option off as well."""
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(H + d)
    M = 7
    n = H * d + G * d + G * dv
    n_pad = (n + 7) // 8 * 8
    proj = torch.randn(M, n_pad, generator=g)
    bv, wq, wk = torch.randn(n, generator=g), torch.rand(H * d, generator=g) + 0.5, torch.rand(G * d, generator=g) + 0.5
    pos = [0, 1, 2, 17, 600, 4999, 5000]
    rates, mag = O.rates_of({"dims": 2 * n_rot, "base": 300.0, "scaling": {"factor": 6.0, "original": 40, "fast": 8.0, "slow": 0.5}})
    q = torch.zeros(M, H * d, device="cuda")
    kc, vc = torch.full((2, G, 5001, d), 5.0, device="cuda"), torch.full((2, G, 5001, dv), 5.0, device="cuda")
    ops.row_attn_prep(proj.cuda(), 0, H * d, (H + G) * d, bv.cuda() if bias else None, wq.cuda() if normed else None,
                      wk.cuda() if normed else None, 1e-3, torch.tensor(rates, dtype=torch.float32, device="cuda") if rates else None, n_rot,
                      mag, pairs, 0.3, q, kc, vc, torch.ones(M, **I32), torch.tensor(pos, **I32), H, G, d, dv)
    p = proj[:, :n].double() + (bv.double() if bias else 0.0)
    qd, kd, vd = p[:, :H * d], p[:, H * d:(H + G) * d], p[:, (H + G) * d:]
    if normed:
        qd, kd = O.rms_unit(qd, 1e-3) * wq.double(), O.rms_unit(kd, 1e-3) * wk.double()
    turn = O.rotate_pairs if pairs else O.rotate_halves

    def at(u):
        full = torch.zeros(5001, *u.shape[1:], dtype=torch.float64)
        full[pos] = u
        return turn(full, rates, mag)[pos] if rates else u

    wantq, wantk = at(qd.view(M, H, d)) * 0.3, at(kd.view(M, G, d))
    assert (q.cpu().double().view(M, H, d) - wantq).abs().max() < 1e-3            # the angle is a float32 product: 5000 * rate
    assert (kc[1, :, pos].cpu().double().transpose(0, 1) - wantk).abs().max() < 3e-3
    assert (vc[1, :, pos].cpu().double().transpose(0, 1) - vd.view(M, G, dv)).abs().max() < 1e-5
    assert float(kc[0].min()) == 5.0 and float(vc[0].min()) == 5.0


# ---- the mixed-score attention kernels: far keys, window edges, tile borders ----------------------------------------------------
def mix_case(T, H, G, d, dv, win, hot=None, dtype=torch.float32, seed=0, boost=30.0, decode=False, sink=True, start=0):
    """mix_attn over T cached positions of one row; tokens start .. T-1 are queries at their own positions (``decode``: one launch
    per token).  A hot pair (query position, key position) gets a raw score far above the rest in head 0, which the mixing hands to
    every head, so that a key that is wrongly masked, skipped or misplaced, and a head that misses another head's scores, shows.
    Returns (got, want, the weight every head gives the hot key)."""
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(seed + T)
    q = torch.randn(T, H, d, generator=g) * 0.3
    k = torch.randn(T, G, d, generator=g) * 0.3
    v = torch.randn(T, G, dv, generator=g)
    if hot is not None:
        u = torch.randn(d, generator=g)
        u = u / u.norm()
        q[hot[0], 0] += boost * u
        k[hot[1], 0] += 3.0 * u
    if dtype != torch.float32:
        q = q.to(dtype).float()            # the 16-bit kernels round the query to the cache's type: give both sides that query
    talk = (torch.eye(H) + torch.randn(H, H, generator=g) * 0.3).to(torch.bfloat16).float()
    talk[:, 0] = talk[:, 0].abs() + 0.5
    snk = torch.randn(H, generator=g) if sink else None
    kc, vc = torch.zeros(2, G, T + 3, d), torch.zeros(2, G, T + 3, dv)
    kc[1, :, :T], vc[1, :, :T] = k.transpose(0, 1), v.transpose(0, 1)
    kc, vc = kc.to(dtype), vc.to(dtype)
    n = T - start
    out = torch.zeros(n, H * dv + 8, dtype=dtype, device="cuda")
    qd, kcd, vcd = q[start:].reshape(n, -1).contiguous().cuda(), kc.cuda(), vc.cuda()
    ws = torch.empty(max(ops.mix_attn_workspace_floats(1, H, dv), 4), device="cuda")
    opt = dict(window=win, workspace=ws, rows=torch.tensor([1], **I32), nb=1)
    sd, td = None if snk is None else snk.cuda(), talk.cuda()
    if decode:
        for i in range(n):
            ops.mix_attn(qd[i:i + 1], kcd, vcd, torch.ones(1, **I32), torch.tensor([start + i], **I32), td, sd, out[i:i + 1, :H * dv], H, G, d, dv,
                         cu=torch.tensor([0, 1], **I32), max_n=1, **opt)
    else:
        ops.mix_attn(qd, kcd, vcd, torch.ones(n, **I32), torch.arange(start, T, **I32), td, sd, out[:, :H * dv], H, G, d, dv,
                     cu=torch.tensor([0, n], **I32), max_n=n, **opt)
    kd, vd = kc[1, :, :T].double().transpose(0, 1), vc[1, :, :T].double().transpose(0, 1)
    want = O.mixed_attention(q.double(), kd, vd, talk.double(), torch.full((H,), -math.inf, dtype=torch.float64) if snk is None else snk.double(),
                             1.0, win)[start:]
    seen = None
    if hot is not None:
        one_hot = torch.zeros(T, G, 1, dtype=torch.float64)
        one_hot[hot[1]] = 1.0
        seen = O.mixed_attention(q.double(), kd, one_hot, talk.double(),
                                 torch.full((H,), -math.inf, dtype=torch.float64) if snk is None else snk.double(), 1.0, win)[hot[0], :, 0]
    assert float(out[:, H * dv:].float().abs().max()) == 0.0          # columns beside the heads are not touched
    return out[:, :H * dv].double().cpu().view(n, H, dv), want, seen


# (tokens, window, hot query, hot key)
EDGES = [(600, 0, 599, 3), (600, 590, 599, 10), (600, 590, 599, 9), (70, 32, 63, 32), (70, 32, 64, 32), (70, 32, 64, 33), (130, 64, 127, 64),
         (130, 64, 128, 64), (130, 65, 128, 64), (97, 96, 95, 0), (97, 96, 96, 0), (40, 1, 7, 6), (40, 1, 7, 7), (1, 4, None, None), (2, 2, 1, 0),
         (3, 2, 2, 0), (200, 40, 199, 160), (200, 40, 199, 159), (300, 33, 290, 258), (300, 33, 290, 257), (129, 128, 128, 1), (65, 0, 64, 0),
         (17, 0, 16, 0), (33, 16, 32, 17), (33, 16, 32, 16)]


def check_case(T, win, hq, hk, tol, **kw):
    got, want, seen = mix_case(T, win=win, hot=None if hq is None else (hq, hk), **kw)
    assert (got - want).abs().max() < tol * max(1.0, float(want.abs().max()))
    if hq is not None:
        visible = 0 <= hq - hk and (win == 0 or hq - hk < win)
        assert (float(seen.min()) > 0.5) if visible else (float(seen.max()) == 0.0)


@pytest.mark.parametrize("T,win,hq,hk", EDGES)
@pytest.mark.parametrize("decode", [False, True])
def test_mixed_attention_far_keys_and_window_edges(T, win, hq, hk, decode):
    for dtype, tol in ((torch.float32, 1e-4), (torch.bfloat16, 3e-2)):
        start = max(0, T - 40) if decode else 0
        check_case(T, win, hq, hk, tol, H=4, G=2, d=24, dv=16, dtype=dtype, decode=decode, start=start)


@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 64, 64), (6, 6, 64, 128), (9, 3, 128, 64), (16, 4, 128, 128), (16, 16, 128, 128), (1, 1, 64, 64),
                                      (24, 4, 64, 64), (32, 8, 128, 128), (18, 9, 64, 128), (32, 16, 128, 64)])
def test_mixed_attention_tile_sizes(H, G, d, dv):
    """Sizes the tensor-core kernel takes, one and two heads per warp, chunks of 32 and of 16 keys: hot pairs across its key chunks
    and query tiles, windows that begin inside a chunk, portions that start in the middle of a sequence, with and without sink."""
    from mlx_parallm_b200._lib import BF16, lib
    plan = lib().b200p_mix_attn_tiles_supported(H, G, d, dv, BF16)
    assert plan // 100 == (1 if H <= 16 else 2) and plan % 100 in (16, 32)
    for k, (T, win, hq, hk) in enumerate(EDGES):
        if T > 1 and hq is not None:
            check_case(T, win, hq, hk, 3e-2, H=H, G=G, d=d, dv=dv, dtype=torch.bfloat16 if k % 3 else torch.float16, seed=k, boost=20.0,
                       sink=k % 2 == 0, start=0 if k % 4 < 2 else min(hq, T // 2))
    for T, win, hq, hk in ((70, 32, 64, 33), (70, 32, 64, 32), (200, 0, 199, 3)):
        check_case(T, win, hq, hk, 3e-2, H=H, G=G, d=d, dv=dv, dtype=torch.bfloat16, boost=20.0, decode=True, start=T - 12)


def test_score_mixing_keeps_32_bits():
    """Mixed scores that cancel: raw scores near 60 whose combination is near one.  A mixing product in 16 bits would be off by a
    tenth; the tile kernel's split product agrees with the per-token kernel to float32 rounding."""
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(1)
    H, G, d, T = 8, 8, 64, 64
    q = torch.randn(T, 1, d, generator=g).expand(T, H, d).to(torch.bfloat16).float() * 4.0
    k = (torch.randn(T, 1, d, generator=g).expand(T, G, d) * 2.0).to(torch.bfloat16)
    v = torch.randn(T, G, 64, generator=g).to(torch.bfloat16)
    talk = torch.zeros(H, H)
    for h in range(H):
        talk[h, h], talk[h, (h + 1) % H] = 1.0, -1.0 + 2.0 ** -5
    kc, vc = k.transpose(0, 1).unsqueeze(0).contiguous().cuda(), v.transpose(0, 1).unsqueeze(0).contiguous().cuda()
    out = torch.zeros(T, H * 64, dtype=torch.bfloat16, device="cuda")
    ops.mix_attn(q.reshape(T, -1).contiguous().cuda(), kc, vc, torch.zeros(T, **I32), torch.arange(T, **I32), talk.cuda(), None, out, H, G, d, 64,
                 cu=torch.tensor([0, T], **I32), rows=torch.zeros(1, **I32), nb=1, max_n=T)
    want = O.mixed_attention(q.double(), k.double(), v.double(), talk.double(), torch.full((H,), -math.inf, dtype=torch.float64), 1.0, 0)
    assert (torch.einsum("thd,shd->ths", q[:, :1], k[:, :1].float()).abs().max()) > 50
    assert (out.double().cpu().view(T, H, 64) - want).abs().max() < 2e-2


@pytest.mark.parametrize("H,G,d,dv,nb", [(8, 2, 64, 64, 5), (16, 1, 64, 32, 3), (4, 4, 128, 128, 40), (6, 3, 128, 64, 150), (3, 1, 10, 6, 9),
                                         (32, 8, 128, 128, 32)])
def test_mixed_attention_decode_batches(H, G, d, dv, nb):
    """Decode steps of many rows of unequal length in one launch (rows out of order, windows that cover all or part of a row)."""
    from mlx_parallm_b200 import ops
    g = torch.Generator().manual_seed(H + nb)
    win = 70
    lens = [int(x) for x in torch.randint(1, 200, (nb,), generator=g)]
    rows = torch.randperm(nb + 2, generator=g)[:nb].tolist()
    Tcap = 256
    talk = (torch.eye(H) + torch.randn(H, H, generator=g) * 0.3).to(torch.bfloat16).float()
    sink = torch.randn(H, generator=g)
    for dtype, tol in ((torch.float32, 1e-4), (torch.bfloat16, 3e-2)):
        kc, vc = torch.zeros(nb + 2, G, Tcap, d), torch.zeros(nb + 2, G, Tcap, dv)
        q = (torch.randn(nb, H, d, generator=g) * 0.3).to(dtype).float()
        for r, n in zip(rows, lens):
            kc[r, :, :n], vc[r, :, :n] = torch.randn(G, n, d, generator=g) * 0.6, torch.randn(G, n, dv, generator=g)
        kc, vc = kc.to(dtype), vc.to(dtype)
        out = torch.zeros(nb, H * dv, dtype=dtype, device="cuda")
        ws = torch.empty(max(ops.mix_attn_workspace_floats(nb, H, dv), 4), device="cuda")
        ops.mix_attn(q.reshape(nb, -1).cuda(), kc.cuda(), vc.cuda(), torch.tensor(rows, **I32), torch.tensor([n - 1 for n in lens], **I32),
                     talk.cuda(), sink.cuda(), out, H, G, d, dv, window=win, cu=torch.arange(nb + 1, **I32), rows=torch.tensor(rows, **I32), nb=nb,
                     max_n=1, workspace=ws)
        for e, (r, n) in enumerate(zip(rows, lens)):
            qe = torch.zeros(n, H, d, dtype=torch.float64)
            qe[-1] = q[e].double()
            ref = O.mixed_attention(qe, kc[r, :, :n].double().transpose(0, 1), vc[r, :, :n].double().transpose(0, 1), talk.double(), sink.double(),
                                    1.0, win)[-1]
            assert (out[e].double().cpu().view(H, dv) - ref).abs().max() < tol * max(1.0, float(ref.abs().max())), e


def test_sink_takes_probability_away():
    """A large sink damps every output by the share it takes; one key left in the window shares with the sink alone."""
    got, want, _ = mix_case(20, 4, 2, 64, 64, 1, dtype=torch.bfloat16)
    none, want_none, _ = mix_case(20, 4, 2, 64, 64, 1, dtype=torch.bfloat16, sink=False)
    assert (got - want).abs().max() < 3e-2 and (none - want_none).abs().max() < 3e-2
    assert float((want / want_none).max()) < 0.95 and float((want / want_none).min()) > 0.0


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


@pytest.mark.parametrize("name", list(CONFIGS))
def test_bfloat16_model(name):
    cfg = CONFIGS[name]()
    m, w = build(cfg, seed=3, dtype=torch.bfloat16, gain=0.7)
    t = toks(cfg, 60, 2)
    got = m.forward_ragged([t], m.make_cache(1), want=[list(range(len(t)))])
    want = O.forward(cfg, w, t)
    per_pos = sorted(O.logits_error(got[i:i + 1], want[i:i + 1]) for i in range(len(t)))       # rounding flips an expert now and then
    assert per_pos[len(t) // 2] < BF16_TOL and per_pos[-1] < 1.0, per_pos[-3:]


def test_bfloat16_model_on_the_tensor_core_paths():
    """Sizes the tile attention kernels take, groups of experts large enough for the tcgen05 grouped product: a prompt, a ragged
    batch and decode steps through the captured step in bfloat16 against the oracle; positions compared by their typical error."""
    from mlx_parallm_b200 import utils
    cfg = O.make_config([
        O.attention_layer(4, 2, 64, 64, 0.125, 100, 32, scaling=(4.0, 128, 8.0, 1.0), mlp=O.dense_mlp(256)),
        O.latent_layer(8, 32, 32, 32, 64, 96, 0.125, 60, mlp=O.moe_mlp(2, 1, 128)),
        O.attention_layer(20, 2, 64, 128, 0.125, 70, 64, mlp=O.moe_mlp(4, 2, 64)),
        O.attention_layer(3, 3, 128, 128, 0.09, 4096, 16),
    ], vocab=200, width=128)
    m, w = build(cfg, seed=7, dtype=torch.bfloat16, gain=0.8)
    t = toks(cfg, 330, 3)
    want = O.forward(cfg, w, t)
    got = m.forward_ragged([t[:300]], m.make_cache(1), want=[list(range(300))])
    per_pos = sorted(O.logits_error(got[i:i + 1], want[i:i + 1]) for i in range(300))
    assert per_pos[150] < BF16_TOL and per_pos[-1] < 1.0, per_pos[-3:]
    lens = [300, 70, 5]
    cache = utils._kv_pool.get_for(m, 3)
    first = m.forward_ragged([t[:n] for n in lens], cache, rows=[2, 0, 1])
    errs = [O.logits_error(first[i:i + 1], want[n - 1:n]) for i, n in enumerate(lens)]
    st = utils._decode_step_for(m, cache, 3, False)
    st.set_rows([2, 0, 1])
    for k in range(30):
        st.tok.copy_(torch.tensor([t[n + k] for n in lens], dtype=torch.int32))
        st.run()
        errs += [O.logits_error(st.logits[i:i + 1], want[n + k:n + k + 1]) for i, n in enumerate(lens)]
    errs.sort()
    assert errs[len(errs) // 2] < BF16_TOL and errs[-1] < 1.0, errs[-3:]


def test_depth_average_reads_results_before_averaging():
    """Weights that make the averages matter: the last layer reads the embedding output and the first layer's result with large
    weights of either sign and its own result with a small one."""
    cfg = CONFIGS["mixed"]()
    w = O.random_weights(cfg, 5)
    n = len(cfg["layers"])
    w[f"l{n - 1}.dwa"] = torch.tensor([1.5, -2.0] + [0.25] * (n - 2) + [0.5])
    w["l0.dwa"] = torch.tensor([-0.75, 1.25])
    m, _ = build(cfg, weights=w)
    t = toks(cfg, 20, 1)
    want = O.forward(cfg, w, t)
    assert O.logits_error(m.forward_ragged([t], m.make_cache(1), want=[list(range(20))]), want) < F32_TOL
    other = dict(w)
    other["l0.dwa"] = torch.tensor([0.0, 1.0])
    assert O.logits_error(O.forward(cfg, other, t), want) > 1e-2


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


@pytest.mark.parametrize("name", ["mixed", "wide"])
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
    """Four prompts of 1, 2, 17 and 40 tokens in one pass, then decoded together while the short ones end: equal to each
    request alone in a cache of its own, and right against the oracle."""
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
    """The tile kernels over a ragged batch: every request's positions as in a batch of its own, up to 16-bit rounding."""
    cfg = O.make_config([
        O.attention_layer(6, 2, 64, 64, 0.125, 40, 32, mlp=O.dense_mlp(96)),
        O.latent_layer(8, 32, 16, 32, 32, 48, 0.125, 24),
        O.attention_layer(20, 10, 64, 64, 0.125, 33, 16),
    ], vocab=90, width=64)
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
    """A row that held a long sequence is released and takes a new one, alone and beside a row that goes on: the new sequence
    sees no keys and no latents of the old one."""
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
        # and through the decode step: a released row starts a sequence with single tokens
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


@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
def test_far_keys_and_a_window_edge_in_the_model(kind):
    """Inside whole models: a sharp softmax over 520 positions whose last answers change clearly when the first half is withheld,
    in three portions and then token by token; and a windowed layer whose answer changes when a token just inside the window
    changes and does not when one just outside does, in a prompt cut at the edge and in decoding."""
    def layer(win):
        if kind == "attention":
            return O.attention_layer(2, 1, 16, 16, 2.0, win, 8, base=1e4, scaling=(4.0, 64, 8.0, 1.0))
        return O.latent_layer(2, 16, 8, 16, 16, 32, 1.5, win, base=1e4)

    cfg = O.make_config([layer(0)], vocab=40, width=32)
    w = O.random_weights(cfg, 12)
    m, _ = build(cfg, weights=w)
    t = toks(cfg, 520, 3)
    a = O.forward(cfg, w, t)
    assert O.logits_error(O.forward(cfg, w, t[260:])[-10:], a[-10:]) > 1e-2
    cache = m.make_cache(1)
    m.forward_ragged([t[:300]], cache)
    m.forward_ragged([t[300:510]], cache)
    got = torch.cat([m.forward_ragged([[tok]], cache) for tok in t[510:]])
    assert O.logits_error(got, a[-10:]) < F32_TOL
    win = 24
    cfg = O.make_config([layer(win)], vocab=40, width=32)
    w = O.random_weights(cfg, 13)
    m, _ = build(cfg, weights=w)
    t = toks(cfg, 90, 4)
    base = O.forward(cfg, w, t)[-1]
    for pos, seen in ((89 - win + 1, True), (89 - win, False)):
        t2 = list(t)
        t2[pos] = (t[pos] + 1) % 40
        moved = O.logits_error(O.forward(cfg, w, t2)[-1][None], base[None])
        assert (moved > 1e-6) if seen else (moved < 1e-12)
        for cut in (89, 89 - win, 60):
            cache = m.make_cache(1)
            m.forward_ragged([t2[:cut]], cache)
            got = torch.cat([m.forward_ragged([[tok]], cache) for tok in t2[cut:]])[-1:]
            assert O.logits_error(got, O.forward(cfg, w, t2)[-1][None]) < F32_TOL


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
    """The engine's own entry point: left-padded prompts with their lengths, prefill, then the captured decode step feeding
    its own argmax back.  Compared with greedy decoding of the oracle, request by request."""
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

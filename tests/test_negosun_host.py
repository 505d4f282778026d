"""Host-side logic of the Negosun family that needs no GPU: the registry, the configuration's checks, the parameter list, the
per-sequence state's layout, and the oracle's own consistency."""
import math

import pytest
import torch

import negosun_oracle as O


def cfg_small():
    return O.make_config([
        O.layer(4, 2, 8, 6, 0.3, v_mix=False, q_temp=(0.4, 3), mlp=O.moe_mlp(6, 2, 12, (3, 2), shared=10)),
        O.layer(6, 2, 4, 5, 0.4, q_temp=None, mlp=O.moe_mlp(3, 3, 8)),
        O.layer(3, 1, 8, 10, 0.3, q_temp=(0.7, 5)),
        O.layer(2, 2, 8, 8, 0.3, v_mix=False, mlp=O.moe_mlp(4, 1, 8, (2, 1), shared=6)),
        O.layer(2, 2, 6, 5, 0.3),
    ], vocab=20, width=16)


def build(cfg):
    from mlx_parallm_b200.utils import _get_classes
    Model, Args = _get_classes(cfg)
    return Model(Args.from_dict(cfg))


def test_registry_parameters_and_branches():
    from mlx_parallm_b200._lib import UNIT_SETS
    cfg = cfg_small()
    m = build(cfg)
    assert m.model_type == "negosun" and m.block_style == "parallel" and m.supports_ragged and m.dense
    assert m.kernel_units in UNIT_SETS and m.residual_mult == 0.6 and m.logit_cap == 20.0
    held = set(O.random_weights(cfg))
    assert set(m.parameter_names()) == held - {"l1.mix.vmix"}                # the first mixing layer's factor is never read
    assert [x.values for x in m.mixers] == ["own", "first", "blend", "own", "blend"]
    assert [(x.temp_coef, x.temp_every) for x in m.mixers] == [(0.4, 3.0), (0.0, 1.0), (0.7, 5.0), (0.5, 7.0), (0.5, 7.0)]
    assert m.runs[2].mlp is None and m.runs[2].norm2_w_name is None and m.runs[3].norm2_w_name == "l3.norm2"
    ff = m.runs[0].mlp
    assert ff.scoring == "softmax_scores" and ff.groups == (3, 2) and ff.renorm and ff.shared.ff == 10 and ff.top == 2 and ff.ff == 12
    assert m.runs[1].mlp.groups == (1, 1) and m.runs[1].mlp.shared is None


def test_options_that_are_absent_or_null():
    cfg = cfg_small()
    for key in ("logit_softcap", "residual_mult"):
        c = {k: v for k, v in cfg.items() if k != key}
        m = build(c)
        assert (m.logit_cap == 0.0) if key == "logit_softcap" else (m.residual_mult == 1.0)
    assert build(dict(cfg, logit_softcap=None)).logit_cap == 0.0
    mlp = O.moe_mlp(6, 2, 12)
    for groups in (None, {"count": 3, "keep": 3}, {"count": 6, "keep": 2}):
        mlp["router"]["groups"] = groups
        ff = build(O.make_config([O.layer(2, 2, 4, 4, 0.5, mlp=mlp)])).runs[0].mlp
        assert ff.groups == ((groups["count"], groups["keep"]) if groups else (1, 1))
    del mlp["router"]["groups"]
    assert build(O.make_config([O.layer(2, 2, 4, 4, 0.5, mlp=mlp)])).runs[0].mlp.groups == (1, 1)


def test_synthetic_shapes_are_the_models_parameters():
    from mlx_parallm_b200 import synth
    cfg = synth.negosun_config(width=64, ff=96, n_layers=3, heads=8, head_dim=16, experts=8, vocab=50, q_rank=3, window=4)
    m = build(cfg)
    shapes = synth.negosun_shapes(cfg)
    assert shapes == O.shapes(cfg) and set(m.parameter_names()) == set(shapes) - {"l0.mix.vmix"}
    w = synth.negosun_random_weights(cfg)
    assert {k: tuple(v.shape) for k, v in w.items()} == shapes and all(v.dtype == torch.bfloat16 for v in w.values())


def test_state_layout():
    from mlx_parallm_b200.models.base import BatchedKVCache, TokenState
    cache = build(cfg_small()).new_cache(2)
    assert len(cache) == 6 and isinstance(cache[-1], TokenState) and all(isinstance(c, BatchedKVCache) for c in cache[:-1])
    cache[0].ensure_capacity(10, torch.float32, "cpu")
    cache[2].ensure_capacity(10, torch.float32, "cpu")
    assert cache[0].keys.shape == (2, 2, 256, 8) and cache[0].values.shape == (2, 2, 256, 6)
    assert cache[2].keys.shape == (2, 1, 256, 8) and cache[2].values.shape == (2, 1, 256, 10)


def test_config_checks():
    cfg = cfg_small()
    good = cfg["layers"][0]
    with pytest.raises(NotImplementedError):
        build(dict(cfg, layers=[dict(good, type="mamba2")]))
    with pytest.raises(NotImplementedError):
        build(dict(cfg, layers=[dict(good, mlp={"kind": "dense", "ff": 8})]))
    for bad in (O.layer(3, 2, 8, 8, 0.3), O.layer(2, 2, 8, 8, 0.3, q_temp=(0.5, 0)), O.layer(2, 2, 8, 8, 0.3, mlp=O.moe_mlp(6, 7, 8)),
                O.layer(2, 2, 8, 8, 0.3, mlp=O.moe_mlp(6, 2, 8, (4, 2))), O.layer(2, 2, 8, 8, 0.3, mlp=O.moe_mlp(6, 3, 8, (3, 1))),
                O.layer(2, 2, 8, 8, 0.3, mlp=O.moe_mlp(6, 2, 8, (3, 4)))):
        with pytest.raises(ValueError):
            build(dict(cfg, layers=[bad]))
    with pytest.raises(ValueError):                                          # value mixing across unequal numbers of values
        build(dict(cfg, layers=[O.layer(2, 2, 8, 8, 0.3), O.layer(2, 1, 8, 8, 0.3)]))
    build(dict(cfg, layers=[O.layer(2, 2, 8, 8, 0.3), O.layer(2, 1, 8, 8, 0.3, v_mix=False), O.layer(2, 1, 4, 16, 0.3)]))
    for bad in (dict(layers=[]), dict(logit_softcap=-1.0)):
        with pytest.raises(ValueError):
            build(dict(cfg, **bad))


def test_oracle_is_causal_and_matches_single_entries():
    """A prefix gives the prefix's logits; attention, temperature, routing, blending and the layer sum agree with sums written out
    one entry at a time: these hold for any correct statement and guard the oracle itself."""
    cfg = cfg_small()
    w = O.random_weights(cfg, 1)
    t = [3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5]
    taps = []
    full = O.forward(cfg, w, t, tap=lambda i, x: taps.append(x))
    assert (O.forward(cfg, w, t[:6]) - full[:6]).abs().max() < 1e-9 and float(full.abs().max()) < 20.0
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(7, n, 6, generator=g, dtype=O.F64) for n in (4, 2, 2))
    got, i, h = O.causal_attention(q, k, v, 0.5), 5, 2
    e = [math.exp(float(q[i, h] @ k[j, 1]) * 0.5) for j in range(i + 1)]
    assert (got[i, h] - sum(a / sum(e) * v[j, 1] for j, a in enumerate(e))).abs().max() < 1e-12
    temp = O.query_temperature(9, {"coef": 0.5, "every": 4})
    assert temp[:3].tolist() == [1.0] * 3 and temp[3] == 1.0 + 0.5 * math.log(2.0) and temp[6] == temp[3] and temp[7] == 1.0 + 0.5 * math.log(3.0)
    z = torch.tensor([[2.0, -1.0, 1.9, 1.8, 0.0, 1.95]], dtype=O.F64)        # three groups of two; the best two: {0, 1} and {4, 5}
    ids, ws = O.route(z, 3, {"count": 3, "keep": 2})
    assert ids.tolist() == [[0, 5, 4]]
    p = [math.exp(a) for a in (2.0, 1.95, 0.0)]
    assert (ws[0] - torch.tensor([a / sum(p) for a in p], dtype=O.F64)).abs().max() < 1e-12
    P = {n: x.double() for n, x in w.items()}
    x0, eps = P["embed"][t], 1e-5
    y0, _ = O.attention(O.norm(x0, P["l0.norm1"], eps), P, "l0.mix.", cfg["layers"][0]["mixer"], eps)
    x1 = x0 + 0.6 * (P["l0.ls1"] * y0 + P["l0.ls2"] * O.feed_forward(O.norm(x0, P["l0.norm2"], eps), P, "l0.mlp.", cfg["layers"][0]["mlp"]))
    assert (taps[0] - x1).abs().max() < 1e-12
    h1, h2 = O.norm(taps[0], P["l1.norm1"], eps), O.norm(taps[1], P["l2.norm1"], eps)
    first = h1 @ P["l1.mix.v"].T + P["l1.mix.v.b"]
    own = h2 @ P["l2.mix.v"].T + P["l2.mix.v.b"]
    lam = float(P["l2.mix.vmix"])
    _, used = O.attention(h2, P, "l2.mix.", cfg["layers"][2]["mixer"], eps, first)
    assert (used - ((1 - lam) * own + lam * first)).abs().max() < 1e-12
    other = dict(w)
    other["l1.mix.vmix"] = w["l1.mix.vmix"] + 0.3                             # the first mixing layer's factor plays no part
    assert torch.equal(O.forward(cfg, other, t), full)

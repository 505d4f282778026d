"""Host-side logic of the Seradra family that needs no GPU: the registry, the configuration's checks, the parameter list, the
per-sequence state's layout, the rotation rates, the activation's constants, and the oracle's own consistency."""
import math

import pytest
import torch

import seradra_oracle as O


def cfg_small():
    return O.make_config([
        O.attention_layer(4, 2, 8, 6, 0.3, 5, 4, base=100.0, scaling=(4.0, 16, 8.0, 1.0), mlp=O.dense_mlp(12)),
        O.latent_layer(4, 8, 4, 8, 6, 12, 0.3, 7, mlp=O.moe_mlp(3, 2, 8)),
        O.attention_layer(2, 2, 8, 8, 0.3, 9, 8),
    ], vocab=20, width=16)


def test_registry_and_parameter_names():
    from mlx_parallm_b200._lib import UNIT_SETS
    from mlx_parallm_b200.utils import _get_classes
    cfg = cfg_small()
    Model, Args = _get_classes(cfg)
    m = Model(Args.from_dict(cfg))
    assert m.model_type == "seradra" and m.block_style == "postnorm" and m.supports_ragged and m.dense and m.depth_average
    assert m.kernel_units in UNIT_SETS
    assert sorted(m.parameter_names()) == sorted(O.random_weights(cfg).keys())
    att, lat, last = m.mixers
    assert att.window == 5 and len(att.rate_values) == 2 and att.mag > 1.0 and att.has_bias and att.row_norm and att.has_sink and not att.pairs
    assert lat.window == 7 and lat.rot_dim == 4 and lat.row == 32 and lat.mag == 1.0
    assert last.mag == 1.0 and m.runs[-1].mlp is None and m.runs[-1].norm2_w_name is None
    assert m.runs[1].mlp.scoring == "softmax_scores" and m.runs[1].mlp.top == 2 and m.runs[1].mlp.weight_on == "output"


def test_synthetic_shapes_are_the_models_parameters():
    from mlx_parallm_b200 import synth
    from mlx_parallm_b200.utils import _get_classes
    cfg = synth.seradra_config(width=64, ff=96, n_layers=4, heads=4, head_dim=16, q_rank=24, kv_rank=32, window=20, rot_dim=8, experts=4, vocab=50)
    Model, Args = _get_classes(cfg)
    m = Model(Args.from_dict(cfg))
    assert sorted(m.parameter_names()) == sorted(synth.seradra_shapes(cfg)) and synth.seradra_shapes(cfg) == O.shapes(cfg)
    w = synth.seradra_random_weights(cfg)
    assert {k: tuple(v.shape) for k, v in w.items()} == synth.seradra_shapes(cfg) and all(v.dtype == torch.bfloat16 for v in w.values())


def test_state_layout():
    from mlx_parallm_b200.models.base import BatchedKVCache, LatentKVCache, TokenState
    from mlx_parallm_b200.utils import _get_classes
    cfg = cfg_small()
    Model, Args = _get_classes(cfg)
    cache = Model(Args.from_dict(cfg)).new_cache(2)
    assert len(cache) == 4 and isinstance(cache[-1], TokenState)
    assert isinstance(cache[0], BatchedKVCache) and isinstance(cache[1], LatentKVCache) and isinstance(cache[2], BatchedKVCache)
    assert cache[1].rank == 32
    cache[0].ensure_capacity(10, torch.float32, "cpu")
    assert cache[0].keys.shape == (2, 2, 256, 8) and cache[0].values.shape == (2, 2, 256, 6)


def test_config_checks():
    from mlx_parallm_b200.utils import _get_classes
    cfg = cfg_small()
    Model, Args = _get_classes(cfg)
    layers = cfg["layers"]
    with pytest.raises(NotImplementedError):
        Args.from_dict(dict(cfg, layers=[dict(layers[0], type="mamba2")]))
    with pytest.raises(NotImplementedError):
        Args.from_dict(dict(cfg, layers=[dict(layers[0], mlp={"kind": "glu", "ff": 8})]))
    for bad in (O.attention_layer(3, 2, 8, 8, 0.3, 5, 4), O.attention_layer(2, 2, 8, 8, 0.3, 5, 10), O.attention_layer(2, 2, 8, 8, 0.3, 5, 3),
                O.latent_layer(2, 8, 3, 8, 6, 12, 0.3, 4), O.attention_layer(2, 2, 8, 8, 0.3, 5, 4, mlp=O.moe_mlp(3, 4, 8))):
        with pytest.raises(ValueError):
            Args.from_dict(dict(cfg, layers=[bad]))
    with pytest.raises(ValueError):
        Args.from_dict(dict(cfg, layers=[]))


@pytest.mark.parametrize("dims,base,scaling", [(8, 10000.0, None), (16, 5e5, (4.0, 2048, 32.0, 1.0)), (48, 250000.0, (8.0, 4096, 32.0, 1.0)),
                                                (6, 100.0, (2.0, 64, 8.0, 1.0)), (4, 7.0, (3.0, 8, 1.0, 1.0))])
def test_rotation_rates(dims, base, scaling):
    from mlx_parallm_b200.models._sequence import stretched_rates
    sc = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    got, mag = stretched_rates(dims, base, sc)
    want, want_mag = O.rates_of({"dims": dims, "base": base, "scaling": sc})
    assert len(got) == dims // 2 and all(abs(a - b) <= 1e-12 * abs(b) for a, b in zip(got, want)) and mag == pytest.approx(want_mag, rel=1e-15)


def test_activation_constants():
    from mlx_parallm_b200.models._sequence import ActivatedFF
    ff = ActivatedFF(8, 16, "xielu")
    ff.set_xielu(torch.tensor([0.3, -0.8]))
    assert ff.act_constants[0] == pytest.approx(math.log1p(math.exp(0.3)), rel=1e-6)
    assert ff.act_constants[1] == pytest.approx(0.5 + math.log1p(math.exp(-0.8)), rel=1e-6)


def test_oracle_prefix_property_window_sink_and_mixing():
    """The oracle is causal (a prefix gives the prefix's logits), forgets what leaves a window, mixes as written, and its depth
    average with weights (0, .., 0, 1) is the plain stream: these hold for any correct statement and guard the oracle itself."""
    cfg = cfg_small()
    w = O.random_weights(cfg, 1)
    t = [3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5]
    full = O.forward(cfg, w, t)
    assert (O.forward(cfg, w, t[:6]) - full[:6]).abs().max() < 1e-9
    g = torch.Generator().manual_seed(0)
    T, H, G, d = 9, 4, 2, 6
    q, k, v = (torch.randn(T, n, d, generator=g, dtype=O.F64) for n in (H, G, G))
    talk, sink = torch.randn(H, H, generator=g, dtype=O.F64), torch.randn(H, generator=g, dtype=O.F64)
    got = O.mixed_attention(q, k, v, talk, sink, 0.5, 3)
    i, h = 7, 2
    s = []
    for j in (5, 6, 7):
        s.append(sum(float(talk[h, a]) * float(q[i, a] @ k[j, a // 2]) * 0.5 for a in range(H)))
    den = sum(math.exp(x) for x in s) + math.exp(float(sink[h]))
    want = sum(math.exp(x) / den * v[j, h // 2] for x, j in zip(s, (5, 6, 7)))
    assert (got[i, h] - want).abs().max() < 1e-12
    k2, v2 = k.clone(), v.clone()
    k2[:4], v2[:4] = 9.0, 9.0
    b = O.mixed_attention(q, k2, v2, talk, sink, 0.5, 3)
    assert (got[6:] - b[6:]).abs().max() == 0.0 and (got[5] - b[5]).abs().max() > 1e-6
    plain = dict(w)
    for n in range(3):
        plain[f"l{n}.dwa"] = torch.eye(n + 2)[-1]
    taps = []
    O.forward(cfg, plain, t, tap=lambda n, x: taps.append(x))
    P = {a: b_.double() for a, b_ in plain.items()}
    x = O.norm(P["embed"][t], P["embed.norm"], 1e-5)
    x = x + O.norm(O.attention(x, P, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5), P["l0.norm1"], 1e-5)
    x = x + O.norm(O.dense_ff(x, P, "l0.mlp."), P["l0.norm2"], 1e-5)
    assert (taps[0] - x).abs().max() < 1e-12
    z = torch.tensor([-3.0, -1e-5, 0.0, 1e-5, 2.0], dtype=O.F64)
    a = torch.tensor([0.2, -0.4], dtype=O.F64)
    up, dn = math.log1p(math.exp(0.2)), 0.5 + math.log1p(math.exp(-0.4))
    ref = [up * x * x + x / 2 if x > 0 else dn * (math.exp(x) - 1 - x) + x / 2 for x in z.tolist()]
    assert (O.xielu(z, a) - torch.tensor(ref, dtype=O.F64)).abs().max() < 1e-12

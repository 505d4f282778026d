"""Slow float64 statement of the Seradra design, one function per mechanism, whole sequences on the CPU.

Written from the design's equations; shares no code with mlx_parallm_b200 (it does not import it).  Notation: T tokens,
W width, weights ``P[name]`` stored [out, in] and applied as a @ P.T.

The design: a normed embedding; sublayers that read the residual stream itself and are normed on their output only; after every
layer the stream becomes a weighted sum of the embedding output and all layers' results so far; two mixers -- grouped
attention with biased projections, q and k normed as whole rows, half-split rotation of the first dimensions (stretched
frequencies), the heads' scores mixed by a matrix, a sliding window and a sink; and latent attention with a rotated key part
shared by the heads and a sliding window --; a dense feed-forward with a two-parameter activation or a routed one whose
weights are the softmax scores of the chosen experts as they are.
"""
import math

import torch

F64 = torch.float64


# ---- elementwise --------------------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """The layers' norm: the stored weight is an offset from one."""
    return rms_unit(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def xielu(z, act):
    """act = (p, q): softplus(p) z^2 + z / 2 above zero, (1/2 + softplus(q)) (e^z - 1 - z) + z / 2 at and below it."""
    up, dn = softplus(act[0]), 0.5 + softplus(act[1])
    neg = torch.clamp(z, max=0.0)
    return torch.where(z > 0, up * z * z + 0.5 * z, dn * (torch.expm1(neg) - neg) + 0.5 * z)


# ---- rotation -----------------------------------------------------------------------------------------------------------
def rates_of(rot):
    """Angle per position of pair i < dims / 2, and the factor on cos and sin.  f_i = base^(-2i/dims); with
    d(t) = dims ln(original / (2 pi t)) / (2 ln base), lo = max(floor(d(fast)), 0), hi = min(ceil(d(slow)), dims - 1) and
    r_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1): rate_i = r_i f_i / factor + (1 - r_i) f_i; magnitude 0.1 ln(factor) + 1."""
    if not rot or not rot.get("dims"):
        return [], 1.0
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def d(t):
        return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(d(float(sc["fast"]))), 0)
    hi = min(math.ceil(d(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def _cos_sin(T, rates, mag, dims):
    ang = torch.arange(T, dtype=F64).unsqueeze(1) * torch.tensor(rates, dtype=F64).unsqueeze(0)
    shape = [T] + [1] * (dims - 2) + [len(rates)]
    return (torch.cos(ang) * mag).view(shape), (torch.sin(ang) * mag).view(shape)


def rotate_halves(u, rates, mag):
    """u [T, ..., d]: dimension i is paired with i + n (n = len(rates)), both below 2 n; the rest passes."""
    n = len(rates)
    c, s = _cos_sin(u.shape[0], rates, mag, u.dim())
    a, b = u[..., :n], u[..., n:2 * n]
    return torch.cat([a * c - b * s, b * c + a * s, u[..., 2 * n:]], -1)


def rotate_pairs(u, rates, mag):
    """u [T, ..., d]: dimension 2i is paired with 2i + 1."""
    n = len(rates)
    c, s = _cos_sin(u.shape[0], rates, mag, u.dim())
    a, b = u[..., 0:2 * n:2], u[..., 1:2 * n:2]
    out = u.clone()
    out[..., 0:2 * n:2] = a * c - b * s
    out[..., 1:2 * n:2] = b * c + a * s
    return out


# ---- mixers -------------------------------------------------------------------------------------------------------------
def visible(T, window):
    """[T, T] bool: position i sees j with 0 <= i - j < window (window 0: every j <= i)."""
    d = torch.arange(T).unsqueeze(1) - torch.arange(T).unsqueeze(0)
    return (d >= 0) & (d < window) if window else d >= 0


def sink_softmax(s, sink):
    """Softmax over the last dimension of s [H, T, T] whose denominator also holds exp(sink_h)."""
    top = torch.maximum(s.max(-1, keepdim=True).values, sink.view(-1, 1, 1))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink.view(-1, 1, 1) - top))


def mixed_attention(q, k, v, talk, sink, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]: raw scores of every head, then score_h = sum_g talk[h, g] raw_g,
    the window, the softmax with its sink, the values of the head's own key/value head."""
    T, H, _ = q.shape
    G = k.shape[1]
    group = torch.arange(H) // (H // G)
    raw = torch.einsum("thd,shd->hts", q, k[:, group]) * scale
    s = torch.einsum("hg,gts->hts", talk, raw)
    s = s.masked_fill(~visible(T, window), -math.inf)
    return torch.einsum("hts,shd->thd", sink_softmax(s, sink), v[:, group])


def attention(h, P, pre, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    q, k, v = (h @ P[pre + n].T + P[pre + n + ".b"] for n in ("q", "k", "v"))
    q = (rms_unit(q, eps) * P[pre + "q.norm"]).view(T, H, d)
    k = (rms_unit(k, eps) * P[pre + "k.norm"]).view(T, G, d)
    rates, mag = rates_of(m.get("rot"))
    q, k = rotate_halves(q, rates, mag), rotate_halves(k, rates, mag)
    window = int((m.get("mask") or {}).get("size", 0))
    o = mixed_attention(q, k, v.view(T, G, dv), P[pre + "talk"], P[pre + "sink"], m["scale"], window)
    return o.reshape(T, H * dv) @ P[pre + "o"].T


def latent_attention(h, P, pre, m, eps):
    """Queries through a normed latent; keys and values from one normed latent per position, plus one rotated key part that
    all heads share.  Every head: [dim unrotated | rot_dim rotated]; sliding window, ordinary softmax."""
    T = h.shape[0]
    H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = rms_unit(h @ P[pre + "dq"].T, eps) * P[pre + "dq.norm"]
    q = (cq @ P[pre + "uq"].T).view(T, H, dn + dr)
    dkv = h @ P[pre + "dkv"].T
    c = rms_unit(dkv[:, :R], eps) * P[pre + "dkv.norm"]
    rates, mag = rates_of(m["rot"])
    k_rot = rotate_pairs(dkv[:, R:], rates, mag)
    q_rot = rotate_pairs(q[..., dn:], rates, mag)
    k = (c @ P[pre + "uk"].T).view(T, H, dn)
    v = (c @ P[pre + "uv"].T).view(T, H, dv)
    s = (torch.einsum("thd,shd->hts", q[..., :dn], k) + torch.einsum("thd,sd->hts", q_rot, k_rot)) * m["scale"]
    window = int((m.get("mask") or {}).get("size", 0))
    s = s.masked_fill(~visible(T, window), -math.inf)
    o = torch.einsum("hts,shd->thd", torch.softmax(s, -1), v)
    return o.reshape(T, H * dv) @ P[pre + "o"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention}


# ---- feed-forward -------------------------------------------------------------------------------------------------------
def dense_ff(h, P, pre):
    return xielu(h @ P[pre + "up"].T, P[pre + "act"]) @ P[pre + "down"].T


def expert(h, P, pre):
    return (silu(h @ P[pre + "gate"].T) * (h @ P[pre + "up"].T)) @ P[pre + "down"].T


def route(h, P, pre, top):
    """(chosen experts [T, top], their weights): the largest of the softmax over all experts, used as they are."""
    w, ids = torch.topk(torch.softmax(h @ P[pre + "router"].T, -1), int(top), dim=-1)
    return ids, w


def routed_ff(h, P, pre, mlp, chosen=None):
    ids, w = route(h, P, pre, mlp["router"]["top"]) if chosen is None else chosen
    out = torch.zeros(h.shape[0], P[pre + "e0.down"].shape[0], dtype=F64)
    for e in range(int(mlp["router"]["experts"])):
        t, slot = (ids == e).nonzero(as_tuple=True)
        if len(t):
            out[t] += w[t, slot].unsqueeze(1) * expert(h[t], P, f"{pre}e{e}.")
    return out


def feed_forward(h, P, pre, mlp, chosen=None):
    return dense_ff(h, P, pre) if mlp["kind"] == "dense" else routed_ff(h, P, pre, mlp, chosen)


# ---- the model ----------------------------------------------------------------------------------------------------------
def depth_average(xs, weights):
    """sum_j weights[j] X_j over the embedding output and the layers' results so far."""
    return sum(weights[j] * xs[j] for j in range(len(xs)))


def forward(cfg, P, tokens, tap=None, chosen=None):
    """Logits [T, vocab] of one sequence.  ``tap(layer, stream)`` after every layer, its averaging included.  ``chosen``: per
    layer the (experts, weights) to use instead of routing (to compare past a close call)."""
    P = {k: v.to(F64) if v.is_floating_point() else v for k, v in P.items()}
    eps = float(cfg["norm"]["eps"])
    x = norm(P["embed"][torch.as_tensor(tokens, dtype=torch.long)], P["embed.norm"], eps)
    xs = [x]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + norm(MIXERS[L["type"]](x, P, p + "mix.", L["mixer"], eps), P[p + "norm1"], eps)
        if L.get("mlp") is not None:
            x = x + norm(feed_forward(x, P, p + "mlp.", L["mlp"], None if chosen is None else chosen[i]), P[p + "norm2"], eps)
        xs.append(x)
        x = depth_average(xs, P[p + "dwa"])
        if tap is not None:
            tap(i, x)
    return norm(x, P["final.norm"], eps) @ P["head"].T


# ---- small configurations and random weights for the tests ------------------------------------------------------------------
def moe_mlp(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def dense_mlp(ff):
    return {"kind": "dense", "ff": ff}


def _rot(dims, base, scaling):
    rot = {"dims": dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return rot


def attention_layer(heads, kv_heads, dim, vdim, scale, window, rot_dims, base=10000.0, scaling=None, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": window}, "rot": _rot(rot_dims, base, scaling)}, "mlp": mlp}


def latent_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window, base=10000.0, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
                                                  "kv_rank": kv_rank, "scale": scale, "mask": {"size": window},
                                                  "rot": _rot(rot_dim, base, None)}, "mlp": mlp}


def make_config(layers, vocab=40, width=32, eps=1e-5):
    return {"architecture": "Seradra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}


def shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "embed.norm": (W,), "final.norm": (W,), "head": (V, W)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        s[p + "norm1"] = (W,)
        s[p + "dwa"] = (i + 2,)
        H = m["heads"]
        if L["type"] == "attention":
            cq, ck, cv = H * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            for n, c in (("q", cq), ("k", ck), ("v", cv)):
                s[f"{p}mix.{n}"], s[f"{p}mix.{n}.b"] = (c, W), (c,)
            s.update({p + "mix.q.norm": (cq,), p + "mix.k.norm": (ck,), p + "mix.talk": (H, H), p + "mix.sink": (H,),
                      p + "mix.o": (W, H * m["vdim"])})
        else:
            s.update({p + "mix.dq": (m["q_rank"], W), p + "mix.dq.norm": (m["q_rank"],), p + "mix.uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                      p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], W), p + "mix.dkv.norm": (m["kv_rank"],),
                      p + "mix.uk": (H * m["dim"], m["kv_rank"]), p + "mix.uv": (H * m["vdim"], m["kv_rank"]), p + "mix.o": (W, H * m["vdim"])})
        mlp = L.get("mlp")
        if mlp is None:
            continue
        s[p + "norm2"] = (W,)
        if mlp["kind"] == "dense":
            s.update({p + "mlp.up": (mlp["ff"], W), p + "mlp.down": (W, mlp["ff"]), p + "mlp.act": (2,)})
        else:
            ff = mlp["expert"]["ff"]
            for e in range(mlp["router"]["experts"]):
                s.update({f"{p}mlp.e{e}.gate": (ff, W), f"{p}mlp.e{e}.up": (ff, W), f"{p}mlp.e{e}.down": (W, ff)})
            s[p + "mlp.router"] = (mlp["router"]["experts"], W)
    return s


def random_weights(cfg, seed=0, dtype=torch.float32, gain=1.0):
    """Random tensors of every shape, scaled so that each branch moves the stream visibly (``gain`` multiplies the projection
    matrices); values are rounded to bfloat16 (kept in ``dtype``) so that a bfloat16 model holds the same numbers."""
    g = torch.Generator().manual_seed(seed)
    P = {}
    for name, shape in shapes(cfg).items():
        leaf = name.split(".")[-1]
        r = torch.randn(shape, generator=g)
        if leaf in ("norm1", "norm2") or name in ("embed.norm", "final.norm"):
            t = r * 0.3
        elif leaf == "norm":
            t = 1.0 + r * 0.3
        elif leaf == "dwa":
            t = r * 0.25
            t[-1] += 1.0
        elif leaf == "talk":
            t = torch.eye(shape[0]) + r * (0.6 / math.sqrt(shape[0]))
        elif leaf in ("sink", "act"):
            t = r * 0.8
        elif leaf == "b":
            t = r * 0.3
        elif name == "embed":
            t = r
        elif len(shape) == 2:
            t = r * (1.5 * gain / math.sqrt(shape[1]))
            if leaf == "router":
                t = t * 1.5
        else:
            raise KeyError(name)
        P[name] = t.to(torch.bfloat16).to(dtype)
    return P


def logits_error(got, want):
    """Worst position: rms over the vocabulary of the centred difference, relative to the rms of the centred expected row."""
    got, want = got.to(F64).cpu(), want.to(F64).cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().clamp_min(1e-30)).max())

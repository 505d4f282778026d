"""Slow float64 statement of the Negosun design, one function per mechanism, whole sequences on the CPU.

Written from the design's equations; shares no code with mlx_parallm_b200 (it does not import it).  Notation: T tokens,
W width, weights ``P[name]`` stored [out, in] and applied as a @ P.T.

The design: every layer adds a mixer and a feed-forward to the stream at once, each reading a norm of its own of the same stream
and scaled channel by channel, the sum multiplied by one constant; grouped attention without positions in its scores -- biased
projections, q and k normed as whole rows, queries that grow with the logarithm of their position, values blended with those of
the first such layer; routed experts chosen inside the best expert groups (a group counts as its best expert) by a softmax over
all experts, beside a shared expert; a head tied to the embedding whose logits are capped by a tanh.
"""
import math

import torch

F64 = torch.float64


# ---- elementwise --------------------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms_unit(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def cap(z, limit):
    return limit * torch.tanh(z / limit) if limit else z


# ---- attention ------------------------------------------------------------------------------------------------------------
def query_temperature(T, q_temp):
    """[T]: 1 + coef ln(floor((p + 1) / every) + 1) at position p (None: ones)."""
    if not q_temp:
        return torch.ones(T, dtype=F64)
    every = int(q_temp["every"])
    return torch.tensor([1.0 + float(q_temp["coef"]) * math.log((p + 1) // every + 1) for p in range(T)], dtype=F64)


def causal_attention(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    group = torch.arange(H) // (H // G)
    s = torch.einsum("thd,shd->hts", q, k[:, group]) * scale
    s = s.masked_fill(torch.triu(torch.ones(T, T, dtype=torch.bool), 1), -math.inf)
    return torch.einsum("hts,shd->thd", torch.softmax(s, -1), v[:, group])


def blend_values(v, first, lam):
    """Values of a blending layer: ``first`` None means that this layer is the first one and keeps its own."""
    return v if first is None else (1.0 - lam) * v + lam * first


def attention(h, P, pre, m, eps, first=None):
    """(output, values used): ``first`` are the values of the first blending layer (None: no blending here)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    q, k, v = (h @ P[pre + n].T + P[pre + n + ".b"] for n in ("q", "k", "v"))
    q, k = norm(q, P[pre + "q.norm"], eps), norm(k, P[pre + "k.norm"], eps)
    q = q * query_temperature(T, m.get("q_temp")).unsqueeze(1)
    v = blend_values(v, first, P[pre + "vmix"] if first is not None else None)
    o = causal_attention(q.view(T, H, d), k.view(T, G, d), v.view(T, G, dv), m["scale"])
    return o.reshape(T, H * dv) @ P[pre + "o"].T, v


# ---- feed-forward -------------------------------------------------------------------------------------------------------
def expert(h, P, pre):
    return (silu(h @ P[pre + "gate"].T) * (h @ P[pre + "up"].T)) @ P[pre + "down"].T


def open_experts(scores, count, keep):
    """[T, E] bool: experts of the ``keep`` best of ``count`` equal groups of neighbours, a group counting as its best expert."""
    T, E = scores.shape
    best = scores.view(T, count, E // count).max(-1).values
    kept = torch.zeros(T, count, dtype=torch.bool).scatter(1, torch.topk(best, keep, dim=-1).indices, True)
    return kept.repeat_interleave(E // count, dim=1)


def route(logits, top, groups=None):
    """(chosen experts [T, top], their weights): the largest softmax scores over all experts among the open groups, divided by their
    sum."""
    s = torch.softmax(logits, -1)
    count, keep = (int(groups["count"]), int(groups["keep"])) if groups else (1, 1)
    w, ids = torch.topk(s.masked_fill(~open_experts(s, count, keep), -1.0), int(top), dim=-1)
    return ids, w / (w.sum(-1, keepdim=True) + 1e-20)


def feed_forward(h, P, pre, mlp):
    r = mlp["router"]
    ids, w = route(h @ P[pre + "router"].T, r["top"], r.get("groups"))
    out = expert(h, P, pre + "shared.") if mlp.get("shared") else torch.zeros_like(h)
    for e in range(int(r["experts"])):
        t, slot = (ids == e).nonzero(as_tuple=True)
        if len(t):
            out[t] += w[t, slot].unsqueeze(1) * expert(h[t], P, f"{pre}e{e}.")
    return out


# ---- the model ----------------------------------------------------------------------------------------------------------
def forward(cfg, P, tokens, tap=None):
    """Logits [T, vocab] of one sequence.  ``tap(layer, stream)`` after every layer."""
    P = {k: v.to(F64) if v.is_floating_point() else v for k, v in P.items()}
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    x = P["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    first = None
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        blends = bool(m.get("v_mix"))
        y, v = attention(norm(x, P[p + "norm1"], eps), P, p + "mix.", m, eps, first if blends else None)
        if blends and first is None:
            first = v
        add = P[p + "ls1"] * y
        if L.get("mlp") is not None:
            add = add + P[p + "ls2"] * feed_forward(norm(x, P[p + "norm2"], eps), P, p + "mlp.", L["mlp"])
        x = x + mult * add
        if tap is not None:
            tap(i, x)
    return cap(norm(x, P["final.norm"], eps) @ P["embed"].T, cfg.get("logit_softcap"))


# ---- small configurations and random weights for the tests ------------------------------------------------------------------
def moe_mlp(experts, top, ff, groups=(1, 1), shared=0):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]}},
            "shared": {"ff": shared} if shared else None}


def layer(heads, kv_heads, dim, vdim, scale, v_mix=True, q_temp=(0.5, 7), mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix,
                                           "q_temp": {"coef": q_temp[0], "every": q_temp[1]} if q_temp else None}, "mlp": mlp}


def make_config(layers, vocab=40, width=32, eps=1e-5, mult=0.6, softcap=20.0):
    return {"architecture": "Negosun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult,
            "logit_softcap": softcap}


def shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "final.norm": (W,)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        s[p + "norm1"] = s[p + "ls1"] = (W,)
        cq, ck, cv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        for n, c in (("q", cq), ("k", ck), ("v", cv)):
            s[f"{p}mix.{n}"], s[f"{p}mix.{n}.b"] = (c, W), (c,)
        s.update({p + "mix.q.norm": (cq,), p + "mix.k.norm": (ck,), p + "mix.o": (W, m["heads"] * m["vdim"])})
        if m["v_mix"]:
            s[p + "mix.vmix"] = ()
        mlp = L.get("mlp")
        if mlp is None:
            continue
        s[p + "norm2"] = s[p + "ls2"] = (W,)
        parts = [(f"{p}mlp.e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if mlp.get("shared"):
            parts.append((p + "mlp.shared.", mlp["shared"]["ff"]))
        for pre, ff in parts:
            s.update({pre + "gate": (ff, W), pre + "up": (ff, W), pre + "down": (W, ff)})
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
        if leaf in ("norm", "norm1", "norm2", "ls1", "ls2"):
            t = 1.0 + r * 0.3
        elif leaf == "vmix":
            t = torch.tensor(0.45) + 0.2 * torch.tanh(r)
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

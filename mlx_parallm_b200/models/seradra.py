"""Seradra: a decoder whose sublayers read the residual stream itself and are normed on their output, and whose layers read a
weighted sum of everything computed before them.

config.json (``"architecture": "Seradra"``) lists the layers one by one -- ``type``, the mixer's sizes, its feed-forward (or
null) -- and gives every size and constant; tensors are named ``l<i>.<part>``.

    embedding     the token's row, rms-normed
    layer         x <- x + n1(mixer(x)); x <- x + n2(ff(x)), n = rms_norm(x) * (1 + w)     (the stored norm weights are offsets from one)
    depth average what follows layer i reads x <- sum_j dwa_i[j] X_j over the embedding output X_0 and the layers' results X_1 .. X_(i+1)
    attention     grouped heads, biases on q, k, v; q and k normed as whole rows; the first rot.dims dimensions of every head rotated
                  half against half, frequencies stretched for long contexts; the heads' scores mixed by a matrix before the
                  softmax; a sliding window; a sink in the denominator
    latent_attention  queries and keys/values through rms-normed latents, one rotated key part shared by all heads (interleaved
                  pairs); a sliding window
    feed-forward  dense W_down act(W_up x) with a two-parameter activation (softplus(p) z^2 + z / 2 above zero,
                  (1/2 + softplus(q)) (e^z - 1 - z) + z / 2 below), or routed experts (silu gate): the ``top`` largest of the softmax
                  over all experts, those scores their weights as they are
    output        the model's norm, the head

The reference has no such graph; the blocks are in models/_sequence.py and run on the ragged-batch kernels of the library.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List

import torch

from ._sequence import (ActivatedFF, GatedFF, HashedBigramEmbedding, HeadMixAttention, LatentAttention, LayerRun, Linear, RoutedExperts,
                        SequenceModel, stretched_rates)
from .base import BaseModelArgs

MIXER_TYPES = ("attention", "latent_attention")


@dataclass
class ModelArgs(BaseModelArgs):
    vocab: int
    width: int
    layers: List[Dict[str, Any]]
    norm: Dict[str, Any] = field(default_factory=dict)
    architecture: str = "Seradra"
    model_type: str = "seradra"

    def __post_init__(self):
        if not self.layers:
            raise ValueError("config 'layers' is empty")
        for i, L in enumerate(self.layers):
            if L.get("type") not in MIXER_TYPES:
                raise NotImplementedError(f"layer {i}: mixer type {L.get('type')!r} is not part of this design")
            m = L["mixer"]
            rot = m.get("rot") or {}
            dims = int(rot.get("dims", 0))
            if L["type"] == "attention":
                if m["heads"] % m.get("kv_heads", m["heads"]):
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                if dims % 2 or dims > int(m["dim"]):
                    raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
            else:
                dr = int(m.get("rot_dim", 0))
                if dr % 2 or (dr and int(rot.get("dims", dr)) != dr):
                    raise ValueError(f"layer {i}: the rotated part has an even size and is rotated whole (rot.dims == rot_dim)")
            mlp = L.get("mlp")
            if mlp is None:
                continue
            if mlp.get("kind") not in ("dense", "moe"):
                raise NotImplementedError(f"layer {i}: feed-forward kind {mlp.get('kind')!r} is not part of this design")
            if mlp["kind"] == "moe" and not (1 <= int(mlp["router"]["top"]) <= int(mlp["router"]["experts"])):
                raise ValueError(f"layer {i}: 1 <= top <= experts")

    @property
    def vocab_size(self) -> int:
        return self.vocab


class Model(SequenceModel):
    block_style = "postnorm"
    kernel_units = "sequence_post"

    def __init__(self, args: ModelArgs):
        super().__init__(args)
        W = args.width
        self.eps = float(args.norm.get("eps", 1e-6))
        self.depth_average = True
        self.embed = HashedBigramEmbedding(args.vocab, W, 1.0)
        for i, L in enumerate(args.layers):
            m = L["mixer"]
            rot = m.get("rot") or {}
            window = int((m.get("mask") or {}).get("size", 0))
            if L["type"] == "attention":
                rates, mag = stretched_rates(int(rot["dims"]), float(rot["base"]), rot.get("scaling")) if rot.get("dims") else ([], 1.0)
                mixer = HeadMixAttention(W, m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"], float(m["scale"]), self.eps,
                                         rates=rates, mag=mag, window=window)
            else:
                dr = int(m.get("rot_dim", 0))
                rates, mag = stretched_rates(dr, float(rot["base"]), rot.get("scaling")) if dr else ([], 1.0)
                mixer = LatentAttention(W, m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], float(m["scale"]), window, self.eps,
                                        rot_dim=dr, rates=rates, mag=mag)
            mlp = L.get("mlp")
            if mlp is None:
                ff = None
            elif mlp["kind"] == "dense":
                ff = ActivatedFF(W, int(mlp["ff"]), "xielu")
            else:
                ff = RoutedExperts(W, int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]), "silu",
                                   router_bias=False, scoring="softmax_scores")
            self.runs.append(LayerRun(i, i, mixer, ff, f"l{i}.norm1", False, f"l{i}.norm2" if ff is not None else None))
        self.mixers = [r.mixer for r in self.runs]
        self.lm_head = Linear(W, args.vocab)

    # -- parameters ------------------------------------------------------------------------------------------
    def parameter_names(self) -> List[str]:
        names = ["embed", "embed.norm", "final.norm", "head"]
        for i, L in enumerate(self.args.layers):
            p = f"l{i}."
            names += [p + "norm1", p + "dwa"]
            if L["type"] == "attention":
                names += [p + "mix." + n for n in ("q", "q.b", "k", "k.b", "v", "v.b", "q.norm", "k.norm", "talk", "sink", "o")]
            else:
                names += [p + "mix." + n for n in ("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "o")]
            mlp = L.get("mlp")
            if mlp is None:
                continue
            names.append(p + "norm2")
            if mlp["kind"] == "dense":
                names += [p + "mlp.up", p + "mlp.down", p + "mlp.act"]
            else:
                for e in range(int(mlp["router"]["experts"])):
                    names += [f"{p}mlp.e{e}.{n}" for n in ("gate", "up", "down")]
                names.append(p + "mlp.router")
        return names

    def load_weights(self, weights: Dict[str, torch.Tensor], device="cuda", strict: bool = True, dtype=None):
        """Matrices go to the device in ``dtype`` (default: as stored); vectors (norms, biases, sinks, depth averages) as float32, the
        layer norms' weights with their one added; the score-mixing matrix is rounded to ``dtype`` and kept as float32.  Projections
        that read the same input are stacked into one matrix, gate / up rows interleaved for the fused epilogue, the experts
        stacked per layer, W_uk stored per head transposed; the rotation's rates are computed on the host in float64."""
        device = torch.device(device)
        missing = [n for n in self.parameter_names() if n not in weights]
        if missing:
            raise KeyError(f"missing parameters: {missing[:4]}{'...' if len(missing) > 4 else ''}")
        if dtype is None:
            dtype = weights["embed"].dtype
        if dtype not in (torch.float32, torch.bfloat16, torch.float16):
            raise TypeError(f"unsupported storage dtype {dtype}")
        self.dtype, self.device = dtype, device
        a, W = self.args, self.args.width

        def put(t):
            return t.to(device=device, dtype=dtype).contiguous()

        def check(name, shape):
            if tuple(weights[name].shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(weights[name].shape)} does not match the config ({tuple(shape)})")

        def vec(name, shape, one_plus=False):
            check(name, shape)
            t = weights[name].float()
            return ((1.0 + t) if one_plus else t).to(device).contiguous()

        def rates(m):
            return torch.tensor(m.rate_values, dtype=torch.float32, device=device) if m.rate_values else None

        check("embed", (a.vocab, W))
        check("head", (a.vocab, W))
        self.embed.weight, self.lm_head.weight = put(weights["embed"]), put(weights["head"])
        self.embed_norm_w = vec("embed.norm", (W,), one_plus=True)
        self.final_norm_w = vec("final.norm", (W,), one_plus=True)
        for r in self.runs:
            i, m = r.layer, r.mixer
            p = f"l{i}.mix."
            r.norm_w = vec(f"l{i}.norm1", (W,), one_plus=True)
            r.avg_w = vec(f"l{i}.dwa", (i + 2,))
            if isinstance(m, HeadMixAttention):
                sizes = {"q": m.col_k, "k": m.col_v - m.col_k, "v": m.n_proj - m.col_v}
                for n, rows in sizes.items():
                    check(p + n, (rows, W))
                check(p + "o", (W, m.n_mix))
                m.in_proj.weight = put(torch.cat([weights[p + n] for n in sizes], 0))
                m.bias = torch.cat([vec(f"{p}{n}.b", (rows,)) for n, rows in sizes.items()], 0).contiguous()
                m.q_norm_w, m.k_norm_w = vec(p + "q.norm", (sizes["q"],)), vec(p + "k.norm", (sizes["k"],))
                check(p + "talk", (m.heads, m.heads))
                m.talk = put(weights[p + "talk"]).float().contiguous()
                m.sink = vec(p + "sink", (m.heads,))
                m.o_proj.weight = put(weights[p + "o"])
                m.rates = rates(m)
            else:
                H, dk, dr, dv, R = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
                check(p + "dq", (m.q_rank, W))
                check(p + "dkv", (R + dr, W))
                check(p + "uq", (H * (dk + dr), m.q_rank))
                check(p + "uk", (H * dk, R))
                check(p + "uv", (H * dv, R))
                check(p + "o", (W, H * dv))
                m.down.weight = put(torch.cat([weights[p + "dq"], weights[p + "dkv"]], 0))
                m.uq.weight = put(weights[p + "uq"])
                m.uk_t = put(weights[p + "uk"].reshape(H, dk, R).transpose(1, 2))          # [H, R, dk]
                m.uv = put(weights[p + "uv"])
                m.o_proj.weight = put(weights[p + "o"])
                m.q_norm_w, m.kv_norm_w = vec(p + "dq.norm", (m.q_rank,)), vec(p + "dkv.norm", (R,))
                m.rates = rates(m)
            ff = r.mlp
            if ff is None:
                continue
            r.norm2_w = vec(f"l{i}.norm2", (W,), one_plus=True)
            q = f"l{i}.mlp."
            if isinstance(ff, ActivatedFF):
                check(q + "up", (ff.ff, W))
                check(q + "down", (W, ff.ff))
                check(q + "act", (2,))
                ff.up.weight, ff.down.weight = put(weights[q + "up"]), put(weights[q + "down"])
                ff.set_xielu(weights[q + "act"])
            else:
                check(q + "router", (ff.experts, W))
                ff.router.weight = put(weights[q + "router"])
                for e in range(ff.experts):
                    check(f"{q}e{e}.gate", (ff.ff, W))
                    check(f"{q}e{e}.up", (ff.ff, W))
                    check(f"{q}e{e}.down", (W, ff.ff))
                ff.gate_up = put(torch.stack([GatedFF.interleave(weights[f"{q}e{e}.gate"], weights[f"{q}e{e}.up"]) for e in range(ff.experts)], 0))
                ff.down = put(torch.stack([weights[f"{q}e{e}.down"] for e in range(ff.experts)], 0))
        self._arenas.clear()
        return self

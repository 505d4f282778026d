"""Negosun: a decoder whose layers add attention and routed experts side by side, each branch behind a norm of its own.

config.json (``"architecture": "Negosun"``) lists the layers one by one -- ``type``, the mixer's sizes, its feed-forward (or
null) -- and gives every size and constant; tensors are named ``l<i>.<part>``.

    layer         x <- x + m (ls1 mixer(n1(x)) + ls2 ff(n2(x))): both branches read the same x, n1 / n2 are rms norms, ls1 / ls2 scale
                  channel by channel, m is ``residual_mult``
    attention     grouped heads, biases on q, k, v; q and k normed as whole rows; no rotation: q at position p is multiplied by
                  1 + coef ln(floor((p + 1) / every) + 1); layers with ``v_mix`` blend their values with those of the first such
                  layer, v <- (1 - lambda) v + lambda v_first, before they are cached
    feed-forward  routed experts (silu gate): softmax over all experts, the ``top`` largest among the experts of the best groups (a
                  group counts as its best expert), their scores over their sum; plus a shared expert
    output        the model's norm, the embedding table as head, logits <- cap tanh(logits / cap)

The reference has no such graph; the blocks are in models/_sequence.py and run on the ragged-batch kernels of the library.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

import torch

from ._sequence import GatedFF, HashedBigramEmbedding, LayerRun, Linear, RoutedExperts, RowNormAttention, SequenceModel
from .base import BaseModelArgs


@dataclass
class ModelArgs(BaseModelArgs):
    vocab: int
    width: int
    layers: List[Dict[str, Any]]
    norm: Dict[str, Any] = field(default_factory=dict)
    residual_mult: float = 1.0
    logit_softcap: Optional[float] = None
    architecture: str = "Negosun"
    model_type: str = "negosun"

    def __post_init__(self):
        if not self.layers:
            raise ValueError("config 'layers' is empty")
        if self.logit_softcap is not None and float(self.logit_softcap) < 0:
            raise ValueError("logit_softcap must be positive (or absent)")
        mixed = None
        for i, L in enumerate(self.layers):
            if L.get("type") != "attention":
                raise NotImplementedError(f"layer {i}: mixer type {L.get('type')!r} is not part of this design")
            m = L["mixer"]
            kv = m.get("kv_heads", m["heads"])
            if m["heads"] % kv:
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if m.get("q_temp") and not float(m["q_temp"]["every"]) > 0:
                raise ValueError(f"layer {i}: q_temp.every must be positive")
            if m.get("v_mix"):
                if mixed is not None and mixed != kv * m["vdim"]:
                    raise ValueError(f"layer {i}: layers that mix values need as many of them as the first one")
                mixed = kv * m["vdim"]
            mlp = L.get("mlp")
            if mlp is None:
                continue
            if mlp.get("kind") != "moe":
                raise NotImplementedError(f"layer {i}: feed-forward kind {mlp.get('kind')!r} is not part of this design")
            r = mlp["router"]
            experts, (count, keep) = int(r["experts"]), expert_groups(r)
            if count < 1 or experts % count or not 1 <= keep <= count or not 1 <= int(r["top"]) <= keep * (experts // count):
                raise ValueError(f"layer {i}: equal expert groups, 1 <= keep <= count, and at least 'top' experts in the kept groups")

    @property
    def vocab_size(self) -> int:
        return self.vocab


def expert_groups(router: Dict[str, Any]) -> tuple:
    """(number of equal groups, groups kept) of a router; without groups all experts form one."""
    g = router.get("groups") or {}
    count = int(g.get("count", 1))
    return count, int(g.get("keep", count))


class Model(SequenceModel):
    block_style = "parallel"
    kernel_units = "sequence_rows"

    def __init__(self, args: ModelArgs):
        super().__init__(args)
        W = args.width
        self.eps = float(args.norm.get("eps", 1e-6))
        self.residual_mult = float(args.residual_mult)
        self.logit_cap = float(args.logit_softcap or 0.0)
        self.embed = HashedBigramEmbedding(args.vocab, W, 1.0)
        first_mixed = next((i for i, L in enumerate(args.layers) if L["mixer"].get("v_mix")), None)
        for i, L in enumerate(args.layers):
            m = L["mixer"]
            qt = m.get("q_temp") or {}
            values = "own" if not m.get("v_mix") else "first" if i == first_mixed else "blend"
            mixer = RowNormAttention(W, m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"], float(m["scale"]), self.eps,
                                     temp_coef=float(qt.get("coef", 0.0)), temp_every=float(qt.get("every", 1)), values=values)
            mlp = L.get("mlp")
            ff = None
            if mlp is not None:
                r = mlp["router"]
                ff = RoutedExperts(W, int(r["experts"]), int(r["top"]), int(mlp["expert"]["ff"]), "silu",
                                   shared_ff=int((mlp.get("shared") or {}).get("ff", 0)), router_bias=False, scoring="softmax_scores",
                                   groups=expert_groups(r), renorm=True)
            self.runs.append(LayerRun(i, i, mixer, ff, f"l{i}.norm1", False, f"l{i}.norm2" if ff is not None else None))
        self.mixers = [r.mixer for r in self.runs]
        self.lm_head = Linear(W, args.vocab)

    # -- parameters ------------------------------------------------------------------------------------------
    def parameter_names(self) -> List[str]:
        """Every tensor that is read (a checkpoint may hold more: the first value-mixing layer's factor is never used)."""
        names = ["embed", "final.norm"]
        for r in self.runs:
            p = f"l{r.layer}."
            names += [p + "norm1", p + "ls1"]
            names += [p + "mix." + n for n in ("q", "q.b", "k", "k.b", "v", "v.b", "q.norm", "k.norm", "o")]
            if r.mixer.values == "blend":
                names.append(p + "mix.vmix")
            if r.mlp is None:
                continue
            names += [p + "norm2", p + "ls2", p + "mlp.router"]
            parts = [f"{p}mlp.e{e}." for e in range(r.mlp.experts)] + ([p + "mlp.shared."] if r.mlp.shared is not None else [])
            names += [pre + n for pre in parts for n in ("gate", "up", "down")]
        return names

    def load_weights(self, weights: Dict[str, torch.Tensor], device="cuda", strict: bool = True, dtype=None):
        """Matrices go to the device in ``dtype`` (default: as stored), the embedding once for both of its uses; vectors (norms,
        biases, channel scales) as float32; the value-mixing factors become launch constants.  q, k and v are one matrix, gate / up
        rows interleaved for the fused epilogue, the experts stacked per layer."""
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

        def vec(name, shape):
            check(name, shape)
            return weights[name].float().to(device).contiguous()

        def glu(prefix, ff):
            check(prefix + "gate", (ff, W))
            check(prefix + "up", (ff, W))
            check(prefix + "down", (W, ff))
            return GatedFF.interleave(weights[prefix + "gate"], weights[prefix + "up"]), weights[prefix + "down"]

        check("embed", (a.vocab, W))
        self.embed.weight = put(weights["embed"])
        self.lm_head.weight = self.embed.weight
        self.final_norm_w = vec("final.norm", (W,))
        for r in self.runs:
            i, m = r.layer, r.mixer
            p = f"l{i}.mix."
            r.norm_w, r.scale1 = vec(f"l{i}.norm1", (W,)), vec(f"l{i}.ls1", (W,))
            sizes = {"q": m.col_k, "k": m.col_v - m.col_k, "v": m.n_proj - m.col_v}
            for n, rows in sizes.items():
                check(p + n, (rows, W))
            check(p + "o", (W, m.n_mix))
            m.in_proj.weight = put(torch.cat([weights[p + n] for n in sizes], 0))
            m.bias = torch.cat([vec(f"{p}{n}.b", (rows,)) for n, rows in sizes.items()], 0).contiguous()
            m.q_norm_w, m.k_norm_w = vec(p + "q.norm", (sizes["q"],)), vec(p + "k.norm", (sizes["k"],))
            m.o_proj.weight = put(weights[p + "o"])
            if m.values == "blend":
                if weights[p + "vmix"].numel() != 1:
                    raise ValueError(f"{p}vmix: one number per layer")
                m.value_mix = float(weights[p + "vmix"])
            ff = r.mlp
            if ff is None:
                continue
            q = f"l{i}.mlp."
            r.norm2_w, r.scale2 = vec(f"l{i}.norm2", (W,)), vec(f"l{i}.ls2", (W,))
            check(q + "router", (ff.experts, W))
            ff.router.weight = put(weights[q + "router"])
            experts = [glu(f"{q}e{e}.", ff.ff) for e in range(ff.experts)]
            ff.gate_up, ff.down = put(torch.stack([e[0] for e in experts], 0)), put(torch.stack([e[1] for e in experts], 0))
            if ff.shared is not None:
                gate_up, down = glu(q + "shared.", ff.shared.ff)
                ff.shared.gate_up.weight, ff.shared.down.weight = put(gate_up), put(down)
        self._arenas.clear()
        return self

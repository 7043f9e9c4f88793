"""Felovik: a decoder whose layers are listed one by one in config.json; every layer has two
mixers side by side, and its norms come after the residual sum.

    {"architecture": "Felovik", "vocab": V, "width": W, "max_positions": P, "norm": {"eps": e},
     "embedding": {"scale": c}, "postln_alpha": a,
     "layers": [{"type": "parallel",
                 "mixer": {"left": {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "scale": s,
                                    "q_temp": {"coef": k, "every": n}},
                           "right": {"heads": H2, "vdim": Dv2, "state": N, "groups": G2,
                                     "conv": taps, "norm_groups": Q}},
                 "mlp": {"kind": "dense", "ff": F, "limit": l}},
                {"type": "parallel", "mixer": {...},
                 "mlp": {"kind": "moe", "expert": {"ff": F},
                         "router": {"experts": E, "top": k,
                                    "groups": {"count": g, "keep": m}}}},
                {"type": "parallel", "mixer": {...}, "mlp": null}]}

The stream starts as the token's embedding times `embedding.scale` plus a learned vector of its
position (`pos`, P rows: sequences are bounded by it). A layer is `x <- norm1(a x + mixer(x)); x
<- norm2(a x + ffn(x))` (`PostNormBlockSpec`) with RMS norms. Its mixer (`ParallelMixerSpec`) is half
the sum of two mixers' outputs, each normed over the width: causal attention without a rotation,
with queries and keys normed a head, queries that grow slowly with their position and an
element-wise output gate (`WindowSinkAttentionSpec` without window and sink), beside the
state-space dual recurrence (`DualScanSpec`). Its feed-forward is dense with clamped branches
(`GatedMLPSpec`), a mixture of gated experts whose router opens the best groups of experts only
(`RoutedExpertsSpec`), or absent. The output head is a matrix of its own. Tensors: `embed`, `pos`,
`l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.left.*`, `l<i>.mix.right.*`, `l<i>.mlp.*`, `final.norm`,
`head`.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .registry import register_architecture
from .specs import (ClampedExpertSpec, ConfigError, DualScanSpec, GatedMLPSpec, LayerCall,
                    ModelSpec, NormSpec, ParallelMixerSpec, PostNormBlockSpec, QueryTemperature,
                    RoutedExpertsSpec, WindowSinkAttentionSpec)

#: the dense feed-forward's activation: y = g * sigmoid(DENSE_ALPHA * g) * (u + 1)
DENSE_ALPHA = 1.702
#: the mixer's output is this times the sum of its two branches' normed outputs
BRANCH_SCALE = 0.5


def _is_int(v) -> bool:
    return isinstance(v, int) and not isinstance(v, bool)


def _is_number(v) -> bool:
    return isinstance(v, (int, float)) and not isinstance(v, bool)


@dataclass(frozen=True)
class FelovikLayer:
    left: dict                      # the attention's own keys, checked
    right: dict                     # the recurrence's
    mlp: Optional[dict]             # None: no feed-forward


@dataclass(frozen=True)
class FelovikConfig:
    vocab: int
    width: int
    max_positions: int
    eps: float
    embed_scale: float
    alpha: float
    layers: tuple
    initializer_range: float = 0.05

    architecture = "Felovik"
    #: the number of learned positions may be left to the table's shape
    needs_tensor_shapes = True

    @classmethod
    def from_dict(cls, raw: dict, tensor_shapes: dict | None = None) -> "FelovikConfig":
        problems = []

        def positive_int(where, holder, key, default=None):
            v = holder.get(key) if isinstance(holder, dict) else None
            if v is None and default is not None:
                return default
            if not _is_int(v) or v <= 0:
                problems.append(f"{where}{key}: expected a positive integer, config.json has {v!r}")
                return 1
            return v

        def number(where, holder, key, low=None):
            v = holder.get(key) if isinstance(holder, dict) else None
            if not _is_number(v) or (low is not None and v <= low):
                problems.append(f"{where}{key}: expected a number"
                                + (f" above {low}" if low is not None else "")
                                + f", config.json has {v!r}")
                return 1.0
            return float(v)

        def holder(where, parent, key, what):
            v = parent.get(key) if isinstance(parent, dict) else None
            if not isinstance(v, dict):
                problems.append(f"{where}{key}: expected an object with {what}")
                return {}
            return v

        vocab = positive_int("", raw, "vocab")
        width = positive_int("", raw, "width")
        rows = (tensor_shapes or {}).get("pos")
        max_positions = positive_int("", raw, "max_positions", rows[0] if rows else None)
        eps = (raw.get("norm") or {}).get("eps")
        if not _is_number(eps) or eps < 0:
            problems.append(f"norm.eps: expected a number >= 0, config.json has {eps!r}")
            eps = 0.0
        embedding = raw.get("embedding")
        embed_scale = 1.0 if embedding is None else number("embedding.", embedding, "scale")
        alpha = number("", raw, "postln_alpha")
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            problems.append("layers: expected a list of layers")
            listed = []
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]."
            if not isinstance(entry, dict) or entry.get("type") != "parallel":
                kind = entry.get("type") if isinstance(entry, dict) else entry
                problems.append(f"{where}type: {kind!r} is not 'parallel'")
                continue
            mixer = holder(where, entry, "mixer", "the two mixers' sizes")
            m, lw = holder(where + "mixer.", mixer, "left", "the attention's sizes"), \
                where + "mixer.left."
            left = {k: positive_int(lw, m, k) for k in ("heads", "dim")}
            left["kv_heads"] = positive_int(lw, m, "kv_heads", left["heads"])
            left["vdim"] = positive_int(lw, m, "vdim", left["dim"])
            left["scale"] = number(lw, m, "scale")
            if left["heads"] % left["kv_heads"]:
                problems.append(f"{lw}{left['heads']} heads are not a multiple of "
                                f"{left['kv_heads']} kv_heads")
            if left["dim"] > 640 or left["vdim"] > 512:
                problems.append(f"{lw}dim up to 640 and vdim up to 512 are what the attention "
                                "kernel takes")
            temp = m.get("q_temp")
            left["q_temp"] = None if temp is None else {
                "coef": number(lw + "q_temp.", temp, "coef"),
                "every": number(lw + "q_temp.", temp, "every", 0)}
            m, rw = holder(where + "mixer.", mixer, "right", "the recurrence's sizes"), \
                where + "mixer.right."
            right = {k: positive_int(rw, m, k) for k in ("heads", "vdim", "state", "conv")}
            right["groups"] = positive_int(rw, m, "groups", 1)
            right["norm_groups"] = positive_int(rw, m, "norm_groups", 1)
            if right["heads"] % right["groups"]:
                problems.append(f"{rw}{right['heads']} heads are not a multiple of "
                                f"{right['groups']} groups")
            if right["heads"] * right["vdim"] % right["norm_groups"]:
                problems.append(f"{rw}heads * vdim is not a multiple of norm_groups "
                                f"{right['norm_groups']}")
            if right["state"] > 256 or right["conv"] > 64:
                problems.append(f"{rw}state up to 256 and conv up to 64 are what the scan kernels "
                                "take")
            if right["heads"] * right["vdim"] > 12000:
                problems.append(f"{rw}heads * vdim up to 12000 is what the gated norm takes")
            mlp = entry.get("mlp")
            if mlp is not None:
                fw = where + "mlp."
                kind = mlp.get("kind") if isinstance(mlp, dict) else mlp
                if kind == "dense":
                    mlp = {"kind": "dense", "ff": positive_int(fw, mlp, "ff"),
                           "limit": number(fw, mlp, "limit", 0.0)}
                elif kind == "moe":
                    r = holder(fw, mlp, "router", "the router's sizes")
                    router = {k: positive_int(fw + "router.", r, k) for k in ("experts", "top")}
                    g = r.get("groups")
                    count = keep = 1
                    if g is not None:
                        count = positive_int(fw + "router.groups.", g, "count")
                        keep = positive_int(fw + "router.groups.", g, "keep")
                        router["groups"] = {"count": count, "keep": keep}
                    if router["experts"] > 1024 or router["top"] > 32:
                        problems.append(f"{fw}router: up to 1024 experts and top up to 32 are what "
                                        "the router kernel takes")
                    if count > 64 or router["experts"] % count or keep > count \
                            or router["experts"] // count * keep < router["top"]:
                        problems.append(f"{fw}router.groups: {count} groups (64 at most, equal) of "
                                        f"which {keep} are kept do not fit {router['experts']} "
                                        f"experts and top {router['top']}")
                    mlp = {"kind": "moe", "router": router,
                           "expert": {"ff": positive_int(fw + "expert.", mlp.get("expert"), "ff")}}
                else:
                    problems.append(f"{fw}kind: {kind!r} is neither 'dense' nor 'moe'")
                    mlp = None
            layers.append(FelovikLayer(left, right, mlp))
        if problems:
            raise ConfigError("config.json cannot describe a Felovik model:\n    "
                              + "\n    ".join(problems))
        return cls(vocab=vocab, width=width, max_positions=max_positions, eps=float(eps),
                   embed_scale=embed_scale, alpha=alpha, layers=tuple(layers),
                   initializer_range=float(raw.get("initializer_range", 0.05)))

    def to_dict(self) -> dict:
        """The config.json that reads back as this configuration."""
        layers = []
        for layer in self.layers:
            left = {k: v for k, v in layer.left.items() if v is not None}
            layers.append({"type": "parallel", "mixer": {"left": left, "right": dict(layer.right)},
                           "mlp": layer.mlp})
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "max_positions": self.max_positions, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embed_scale}, "postln_alpha": self.alpha,
                "layers": layers, "initializer_range": self.initializer_range}

    # -- the parts' descriptions -----------------------------------------------------------

    def _mixer(self, layer, norm):
        a, b = layer.left, layer.right
        temp = a["q_temp"]
        left = WindowSinkAttentionSpec(
            hidden=self.width, heads=a["heads"], kv_heads=a["kv_heads"], head_dim=a["dim"],
            value_dim=a["vdim"], scale=a["scale"], window=None, keep_first=0, eps=self.eps,
            position=None, sink=False, qk_norm="head", bias=False, gate=True,
            q_temp=None if temp is None else QueryTemperature(temp["coef"], temp["every"]))
        right = DualScanSpec(
            hidden=self.width, heads=b["heads"], value_dim=b["vdim"], state=b["state"],
            groups=b["groups"], taps=b["conv"], norm_groups=b["norm_groups"], eps=self.eps)
        return ParallelMixerSpec(hidden=self.width, left=left, right=right, branch_norm=norm,
                                 scale=BRANCH_SCALE)

    def _ffn(self, layer):
        mlp = layer.mlp
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return GatedMLPSpec(hidden=self.width, intermediate=mlp["ff"], activation="clamped",
                                names=("gate", "up", "down"), limit=mlp["limit"],
                                alpha=DENSE_ALPHA, plus=1.0)
        r = mlp["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        return RoutedExpertsSpec(
            hidden=self.width, experts=r["experts"], top=r["top"],
            expert=ClampedExpertSpec(mlp["expert"]["ff"], limit=float("inf"), alpha=1.0, plus=0.0),
            shared=None, shared_gate=False, score="softmax", renormalize=True, weight_input=False,
            groups=groups["count"], keep_groups=groups["keep"])

    def model_spec(self) -> ModelSpec:
        norm = NormSpec(size=self.width, eps=self.eps, suffix="")
        blocks, ignore = [], []
        for i, layer in enumerate(self.layers):
            ffn = self._ffn(layer)
            if ffn is None:        # a checkpoint may still carry the absent sublayer's norm
                ignore.append(f"l{i}.norm2")
            blocks.append(PostNormBlockSpec(prefix=f"l{i}.", mixer=self._mixer(layer, norm),
                                            ffn=ffn, norm=norm, alpha=self.alpha))
        order = tuple(LayerCall(block=i, cache=i) for i in range(len(blocks)))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden=self.width,
            blocks=tuple(blocks), run_order=order, final_norm=norm, tie_head=False,
            max_positions=self.max_positions, embed_name="embed", position_name="pos",
            final_norm_name="final.norm", head_name="head", stored_dtype="bfloat16",
            init_std=self.initializer_range, embed_scale=self.embed_scale,
            ignore_tensors=tuple(ignore))


register_architecture(FelovikConfig.architecture, FelovikConfig)

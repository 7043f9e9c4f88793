"""Gozolix: a decoder whose layers are listed one by one in config.json; a layer's mixer and
feed-forward read the output of one norm and are added to the stream together.

    {"architecture": "Gozolix", "vocab": V, "width": W, "norm": {"eps": e},
     "embedding": {"scale": c, "bigram": {"buckets": B, "mul_prev": a, "mul_cur": b}},
     "layers": [{"type": "delta",
                 "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "conv": taps},
                 "mlp": {"kind": "dense", "ff": F}},
                {"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": Dv, "scale": s,
                           "softcap": t, "q_temp": {"coef": k, "every": n}},
                 "mlp": {"kind": "moe", "expert": {"ff": F}, "shared": {"ff": F2},
                         "router": {"experts": E, "top": k, "scale": r,
                                    "groups": {"count": g, "keep": m}}}},
                {"type": "attention", "mixer": {..., "kv_from": 1}, "mlp": null}]}

The stream starts as the token's embedding times `embedding.scale` plus a row of a table of pairs of
tokens (`BigramSpec`). A layer is `h = norm1(x); x <- x + mixer(h) + ff(h)` (`ParallelBlockSpec`)
with RMS norms. Its mixer is the gated delta rule (`GatedDeltaSpec`) or causal attention without a
rotation, with biases, queries that grow slowly with their position, soft-capped scores and a
penalty that grows linearly with the distance (`WindowSinkAttentionSpec` without window and sink);
with `kv_from` an attention layer uses an earlier attention layer's cached keys and values (its
layer call names that layer's cache entry). Its feed-forward is dense with the square of relu
(`DenseMLPSpec`), a mixture of gated experts with a shared one, whose router opens the best groups
of experts only (`RoutedExpertsSpec`), or absent. The output head is a matrix of its own. Tensors:
`embed`, `bigram`, `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm`, `head`.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .registry import register_architecture
from .specs import (BigramSpec, ClampedExpertSpec, ConfigError, DenseMLPSpec, GatedDeltaSpec,
                    LayerCall, ModelSpec, NormSpec, ParallelBlockSpec, QueryTemperature,
                    RoutedExpertsSpec, WindowSinkAttentionSpec)

#: inside the root of a unit vector of the delta rule
UNIT_EPS = 1e-6
#: a head's distance penalty is 2 ** (-SLOPE_SPAN * (h + 1) / heads)
SLOPE_SPAN = 8.0
#: the experts of a group whose scores are summed to the group's
GROUP_TOP = 2
#: the design has no table of positions; this bounds a sequence only through the cache
MAX_POSITIONS = 1 << 22


def head_slopes(heads: int) -> tuple:
    return tuple(2.0 ** (-SLOPE_SPAN * (h + 1) / heads) for h in range(heads))


def _is_int(v) -> bool:
    return isinstance(v, int) and not isinstance(v, bool)


def _is_number(v) -> bool:
    return isinstance(v, (int, float)) and not isinstance(v, bool)


@dataclass(frozen=True)
class GozolixLayer:
    type: str                       # "delta" | "attention"
    mixer: dict                     # the mixer's own keys, checked
    mlp: Optional[dict]             # None: no feed-forward


@dataclass(frozen=True)
class GozolixConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    bigram: Optional[dict]          # None: no table of pairs
    layers: tuple
    initializer_range: float = 0.05

    architecture = "Gozolix"

    @classmethod
    def from_dict(cls, raw: dict) -> "GozolixConfig":
        problems = []

        def integer(where, holder, key, default=None, low=1):
            v = holder.get(key) if isinstance(holder, dict) else None
            if v is None and default is not None:
                return default
            if not _is_int(v) or v < low:
                problems.append(f"{where}{key}: expected an integer of at least {low}, config.json "
                                f"has {v!r}")
                return max(low, 1)
            return v

        def number(where, holder, key, low=None, default=None):
            v = holder.get(key) if isinstance(holder, dict) else None
            if v is None and default is not None:
                return default
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

        def heads_of(where, m):
            out = {k: integer(where, m, k) for k in ("heads", "dim")}
            out["kv_heads"] = integer(where, m, "kv_heads", out["heads"])
            out["vdim"] = integer(where, m, "vdim", out["dim"])
            if out["heads"] % out["kv_heads"]:
                problems.append(f"{where}{out['heads']} heads are not a multiple of "
                                f"{out['kv_heads']} kv_heads")
            return out

        vocab = integer("", raw, "vocab")
        width = integer("", raw, "width")
        eps = (raw.get("norm") or {}).get("eps")
        if not _is_number(eps) or eps < 0:
            problems.append(f"norm.eps: expected a number >= 0, config.json has {eps!r}")
            eps = 0.0
        embedding = raw.get("embedding") or {}
        embed_scale = number("embedding.", embedding, "scale", default=1.0)
        bigram = embedding.get("bigram") if isinstance(embedding, dict) else None
        if bigram is not None:
            where = "embedding.bigram."
            bigram = {"buckets": integer(where, bigram, "buckets"),
                      "mul_prev": integer(where, bigram, "mul_prev", low=0),
                      "mul_cur": integer(where, bigram, "mul_cur", low=0)}
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            problems.append("layers: expected a list of layers")
            listed = []
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]."
            kind = entry.get("type") if isinstance(entry, dict) else entry
            mw = where + "mixer."
            if kind == "delta":
                m = holder(where, entry, "mixer", "the recurrence's sizes")
                mixer = heads_of(mw, m)
                mixer["conv"] = integer(mw, m, "conv")
                if mixer["dim"] > 512 or mixer["conv"] > 64:
                    problems.append(f"{mw}dim up to 512 and conv up to 64 are what the delta "
                                    "kernels take")
            elif kind == "attention":
                m = holder(where, entry, "mixer", "the attention's sizes")
                mixer = heads_of(mw, m)
                mixer["scale"] = number(mw, m, "scale")
                mixer["softcap"] = None if m.get("softcap") is None else number(mw, m, "softcap", 0)
                if mixer["dim"] > 640 or mixer["vdim"] > 512:
                    problems.append(f"{mw}dim up to 640 and vdim up to 512 are what the attention "
                                    "kernel takes")
                temp = m.get("q_temp")
                mixer["q_temp"] = None if temp is None else {
                    "coef": number(mw + "q_temp.", temp, "coef"),
                    "every": number(mw + "q_temp.", temp, "every", 0)}
                mixer["kv_from"] = source = m.get("kv_from")
                if source is not None:
                    other = layers[source] if _is_int(source) and 0 <= source < len(layers) else None
                    if other is None or other.type != "attention" \
                            or other.mixer["kv_from"] is not None:
                        problems.append(f"{mw}kv_from: {source!r} is not an earlier attention layer "
                                        "with keys and values of its own")
                    elif any(other.mixer[k] != mixer[k] for k in ("kv_heads", "dim", "vdim")):
                        problems.append(f"{mw}kv_from: layer {source} has other kv_heads, dim or "
                                        "vdim")
            else:
                problems.append(f"{where}type: {kind!r} is neither 'delta' nor 'attention'")
                layers.append(GozolixLayer("", {}, None))       # (layers are named by their place)
                continue
            mlp = entry.get("mlp")
            if mlp is not None:
                fw = where + "mlp."
                kind_ff = mlp.get("kind") if isinstance(mlp, dict) else mlp
                if kind_ff == "dense":
                    mlp = {"kind": "dense", "ff": integer(fw, mlp, "ff")}
                elif kind_ff == "moe":
                    r = holder(fw, mlp, "router", "the router's sizes")
                    rw = fw + "router."
                    router = {k: integer(rw, r, k) for k in ("experts", "top")}
                    router["scale"] = number(rw, r, "scale", default=1.0)
                    g = r.get("groups")
                    count = keep = 1
                    if g is not None:
                        count = integer(rw + "groups.", g, "count")
                        keep = integer(rw + "groups.", g, "keep")
                        router["groups"] = {"count": count, "keep": keep}
                    if router["experts"] > 1024 or router["top"] > 32:
                        problems.append(f"{rw[:-1]}: up to 1024 experts and top up to 32 are what "
                                        "the router kernel takes")
                    if count > 64 or router["experts"] % count or keep > count \
                            or router["experts"] // count * keep < router["top"]:
                        problems.append(f"{rw}groups: {count} groups (64 at most, equal) of which "
                                        f"{keep} are kept do not fit {router['experts']} experts "
                                        f"and top {router['top']}")
                    raw_mlp = mlp
                    mlp = {"kind": "moe", "router": router,
                           "expert": {"ff": integer(fw + "expert.", raw_mlp.get("expert"), "ff")}}
                    if raw_mlp.get("shared") is not None:
                        mlp["shared"] = {"ff": integer(fw + "shared.", raw_mlp["shared"], "ff")}
                else:
                    problems.append(f"{fw}kind: {kind_ff!r} is neither 'dense' nor 'moe'")
                    mlp = None
            layers.append(GozolixLayer(kind, mixer, mlp))
        if problems:
            raise ConfigError("config.json cannot describe a Gozolix model:\n    "
                              + "\n    ".join(problems))
        return cls(vocab=vocab, width=width, eps=float(eps), embed_scale=embed_scale,
                   bigram=bigram, layers=tuple(layers),
                   initializer_range=float(raw.get("initializer_range", 0.05)))

    def to_dict(self) -> dict:
        """The config.json that reads back as this configuration."""
        embedding = {"scale": self.embed_scale}
        if self.bigram is not None:
            embedding["bigram"] = dict(self.bigram)
        layers = [{"type": layer.type,
                   "mixer": {k: v for k, v in layer.mixer.items() if v is not None},
                   "mlp": layer.mlp} for layer in self.layers]
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.eps}, "embedding": embedding, "layers": layers,
                "initializer_range": self.initializer_range}

    # -- the parts' descriptions -----------------------------------------------------------

    def _mixer(self, layer):
        m = layer.mixer
        if layer.type == "delta":
            return GatedDeltaSpec(hidden=self.width, heads=m["heads"], kv_heads=m["kv_heads"],
                                  head_dim=m["dim"], value_dim=m["vdim"], taps=m["conv"],
                                  q_scale=m["dim"] ** -0.5, eps=self.eps, unit_eps=UNIT_EPS)
        temp = m["q_temp"]
        return WindowSinkAttentionSpec(
            hidden=self.width, heads=m["heads"], kv_heads=m["kv_heads"], head_dim=m["dim"],
            value_dim=m["vdim"], scale=m["scale"], window=None, keep_first=0, eps=self.eps,
            position=None, sink=False, qk_norm=None, bias=True, softcap=m["softcap"],
            slopes=head_slopes(m["heads"]), own_kv=m["kv_from"] is None,
            q_temp=None if temp is None else QueryTemperature(temp["coef"], temp["every"]))

    def _ffn(self, layer):
        mlp = layer.mlp
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return DenseMLPSpec(hidden=self.width, intermediate=mlp["ff"],
                                activation="relu_squared")
        r = mlp["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}

        def gated(ff):          # the plain gated silu
            return ClampedExpertSpec(ff, limit=float("inf"), alpha=1.0, plus=0.0)

        return RoutedExpertsSpec(
            hidden=self.width, experts=r["experts"], top=r["top"], expert=gated(mlp["expert"]["ff"]),
            shared=gated(mlp["shared"]["ff"]) if "shared" in mlp else None, shared_gate=False,
            score="sigmoid", renormalize=True, weight_input=False, groups=groups["count"],
            keep_groups=groups["keep"], group_top=GROUP_TOP, scale=r["scale"])

    def model_spec(self) -> ModelSpec:
        norm = NormSpec(size=self.width, eps=self.eps, suffix="")
        blocks, order, entry_of = [], [], {}
        for i, layer in enumerate(self.layers):
            blocks.append(ParallelBlockSpec(prefix=f"l{i}.", mixer=self._mixer(layer),
                                            ffn=self._ffn(layer), norm=norm))
            source = layer.mixer.get("kv_from")
            if source is None:
                entry_of[i] = len(entry_of)
            order.append(LayerCall(block=i, cache=entry_of[i if source is None else source]))
        return ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden=self.width,
            blocks=tuple(blocks), run_order=tuple(order), final_norm=norm, tie_head=False,
            max_positions=MAX_POSITIONS, embed_name="embed", final_norm_name="final.norm",
            head_name="head", stored_dtype="bfloat16", init_std=self.initializer_range,
            embed_scale=self.embed_scale,
            bigram=None if self.bigram is None else BigramSpec("bigram", **self.bigram))


register_architecture(GozolixConfig.architecture, GozolixConfig)

"""Configuration of the Sozudra decoder: layers listed one by one, each either differential attention inside a sliding window
or two mixers side by side (window attention on unit-RMS queries and keys with values that turn with their position, and a
minGRU), and beside it - not behind it - a routed mixture of gated experts with a gated shared expert.  Mixer and
feed-forward read the same float32 stream, each under an RMSNorm of its own.  The embedded tokens get a row per pair of
neighbouring tokens; a span of layers may run several times in a row; the LM head is a tensor of its own.

config.json keys (all sizes and every constant that may differ between models are read, none is assumed):

    architecture            "Sozudra"
    width, vocab            model width and vocabulary size
    norm.eps                eps of every norm
    residual_mult           factor on what a layer adds to the stream
    embedding.bigram        buckets, mul_prev, mul_cur (absent or null: no bigram rows)
    layers[i].type          "parallel" | "attention"
    layers[i].mixer         attention: heads, kv_heads, dim, vdim, scale, diff, softcap (absent: no cap), mask.size (absent: every
                                       earlier key), rot.{dims, base, scaling (absent: none): {factor, original, fast, slow}}
                            parallel: left (as attention, without diff), right.width, left_scale, right_scale
    layers[i].mlp           null | {"kind": "moe", "expert": {"ff": n}, "router": {"experts": E, "top": k}, "shared": {"ff": m} | null}
    loop                    {start, stop, times}: layers start .. stop - 1 run `times` times in a row (absent or null: once)
    max_positions           optional: the longest sequence the rotation tables are ever built for

Tensor names: embed, bigram, head, final.norm, l<i>.norm1, l<i>.norm2, l<i>.mix.{q, q.b, k, k.b, v, v.b, lq1, lk1, lq2, lk2, o} |
l<i>.mix.left.{q, k, v, o} and l<i>.mix.right.{z, z.b, x, x.b, g, o}, l<i>.mlp.{router, router.b, e<j>.gate, e<j>.up, e<j>.down,
shared.gate, shared.up, shared.down, shared.sg}.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from ..errors import ConfigError
from .reader import NumberReader, is_int
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

DEFAULT_MAX_POSITIONS = 1 << 17       # the design sets no limit; the engine's tables are built for max_model_len
MIXERS = ("parallel", "attention")
SCALING = ("factor", "original", "fast", "slow")


@dataclass(frozen=True)
class SozudraLayer:
    type: str                              # one of MIXERS
    mixer: Dict[str, Any]                  # sizes and constants; an attention's are flat (rot_dims, rot_base, rot_scaling, window, ...)
    mlp: Optional[Dict[str, Any]]          # None | {ff, experts, top, shared_ff | None}


class _Reader(NumberReader):
    """... and this design's mixers and feed-forwards."""

    def attention(self, m, at: str, differential: bool) -> Dict[str, Any]:
        if not isinstance(m, dict):
            self.problems.append(at + "must be an object")
            m = {}
        out: Dict[str, Any] = {key: self.integer(m, key, at) for key in ("heads", "kv_heads", "dim", "vdim")}
        out["scale"] = self.number(m, "scale", at, positive=False)
        if out["heads"] % out["kv_heads"]:
            self.problems.append(at + f"{out['heads']} query heads cannot share {out['kv_heads']} key/value heads")
        if differential:
            out["diff"] = self.number(m, "diff", at, positive=False)
        elif out["vdim"] % 2:
            self.problems.append(at + f"values that turn in pairs need an even `vdim`, got {out['vdim']}")
        cap = m.get("softcap")
        out["softcap"] = None if cap is None else self.number(m, "softcap", at)
        mask = m.get("mask")
        out["window"] = None if mask is None else self.integer(mask, "size", at + "mask: ")
        rot = m.get("rot")
        out["rot_dims"] = self.integer(rot, "dims", at + "rot: ", minimum=2)
        out["rot_base"] = self.number(rot, "base", at + "rot: ")
        if out["rot_dims"] % 2 or out["rot_dims"] > out["dim"]:
            self.problems.append(at + f"`rot.dims` must be even and at most dim = {out['dim']}, got {out['rot_dims']}")
        scaling = rot.get("scaling") if isinstance(rot, dict) else None
        out["rot_scaling"] = None
        if scaling is not None:
            values = tuple(self.number(scaling, key, at + "rot.scaling: ") for key in SCALING)
            if out["rot_base"] == 1.0:
                self.problems.append(at + "rot.scaling: a base of 1 gives every pair the same frequency")
            out["rot_scaling"] = values
        return out

    def moe(self, raw, at: str) -> Optional[Dict[str, Any]]:
        if raw is None:
            return None
        if not isinstance(raw, dict) or raw.get("kind") != "moe":
            self.problems.append(at + f"`mlp` must be null or an object of kind \"moe\", got {raw!r}")
            return None
        router = raw.get("router")
        mlp = {"ff": self.integer(raw.get("expert"), "ff", at + "mlp.expert: "),
               "experts": self.integer(router, "experts", at + "mlp.router: "),
               "top": self.integer(router, "top", at + "mlp.router: "), "shared_ff": None}
        if mlp["top"] > mlp["experts"]:
            self.problems.append(at + f"mlp.router: `top` {mlp['top']} exceeds `experts` {mlp['experts']}")
        if raw.get("shared") is not None:
            mlp["shared_ff"] = self.integer(raw.get("shared"), "ff", at + "mlp.shared: ")
        return mlp


@dataclass(frozen=True)
class SozudraConfig:
    width: int
    vocab: int
    eps: float
    residual_mult: float
    bigram: Optional[Tuple[int, int, int]]         # (buckets, mul_prev, mul_cur)
    layers: Tuple[SozudraLayer, ...]
    loop: Optional[Tuple[int, int, int]] = None    # (start, stop, times)
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()
    raw: Dict[str, Any] = field(default_factory=dict, compare=False, repr=False)

    ARCHITECTURE = "Sozudra"

    @property
    def architecture(self) -> str:
        return self.ARCHITECTURE

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    # ---- reading -------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, obj: Dict[str, Any], where: str = "config.json") -> "SozudraConfig":
        r = _Reader()
        p = r.problems
        width = r.integer(obj, "width", "")
        vocab = r.integer(obj, "vocab", "")
        eps = r.number(obj.get("norm"), "eps", "norm: ")
        mult = r.number(obj, "residual_mult", "", positive=False)
        bigram = None
        raw_bigram = (obj.get("embedding") or {}).get("bigram") if isinstance(obj.get("embedding") or {}, dict) else None
        if obj.get("embedding") is not None and not isinstance(obj["embedding"], dict):
            p.append(f"`embedding` must be an object, got {obj['embedding']!r}")
        if raw_bigram is not None:
            bigram = (r.integer(raw_bigram, "buckets", "embedding.bigram: "), r.integer(raw_bigram, "mul_prev", "embedding.bigram: ", 0),
                      r.integer(raw_bigram, "mul_cur", "embedding.bigram: ", 0))
        raw_layers = obj.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError(p + ["`layers` must be a non-empty list"], where)
        layers: List[SozudraLayer] = []
        for i, e in enumerate(raw_layers):
            at = f"layers[{i}]: "
            if not isinstance(e, dict):
                p.append(at + "must be an object")
                continue
            kind, m = e.get("type"), e.get("mixer")
            if kind not in MIXERS:
                p.append(at + f"`type` = {kind!r} is not known ({', '.join(MIXERS)})")
                continue
            if kind == "attention":
                mixer = r.attention(m, at, differential=True)
            else:
                m = m if isinstance(m, dict) else {}
                mixer = {"left": r.attention(m.get("left"), at + "left: ", differential=False),
                         "right_width": r.integer(m.get("right"), "width", at + "right: "),
                         "left_scale": r.number(m, "left_scale", at, positive=False),
                         "right_scale": r.number(m, "right_scale", at, positive=False)}
            layers.append(SozudraLayer(kind, mixer, r.moe(e.get("mlp"), at)))
        loop = None
        raw_loop = obj.get("loop")
        if raw_loop is not None:
            start = r.integer(raw_loop, "start", "loop: ", minimum=0)
            stop = r.integer(raw_loop, "stop", "loop: ", minimum=0)
            times = r.integer(raw_loop, "times", "loop: ")
            if not start <= stop <= len(raw_layers):
                p.append(f"loop: start {start} and stop {stop} must name a span of the {len(raw_layers)} layers")
            loop = (start, stop, times)
        max_pos = obj.get("max_positions", DEFAULT_MAX_POSITIONS)
        if not is_int(max_pos) or max_pos < 1:
            p.append(f"`max_positions` must be a positive integer, got {max_pos!r}")
            max_pos = DEFAULT_MAX_POSITIONS
        eos = obj.get("eos_token_id")
        eos_ids: Tuple[int, ...] = ()
        if is_int(eos):
            eos_ids = (eos,)
        elif isinstance(eos, list) and all(is_int(t) for t in eos):
            eos_ids = tuple(eos)
        elif eos is not None:
            p.append(f"`eos_token_id` must be an integer or a list of integers, got {eos!r}")
        if p:
            raise ConfigError(p, where)
        return cls(width=width, vocab=vocab, eps=eps, residual_mult=mult, bigram=bigram, layers=tuple(layers), loop=loop,
                   max_positions=max_pos, eos_token_ids=eos_ids, raw=dict(obj))

    # ---- writing -------------------------------------------------------------------------------
    @staticmethod
    def _attention_dict(flat: Dict[str, Any]) -> Dict[str, Any]:
        m = dict(flat)
        rot = {"dims": m.pop("rot_dims"), "base": m.pop("rot_base")}
        scaling, window = m.pop("rot_scaling"), m.pop("window")
        if scaling is not None:
            rot["scaling"] = dict(zip(SCALING, scaling))
        m["rot"] = rot
        if window is not None:
            m["mask"] = {"size": window}
        if m["softcap"] is None:
            del m["softcap"]
        return m

    def to_dict(self) -> Dict[str, Any]:
        out_layers = []
        for layer in self.layers:
            m = layer.mixer
            if layer.type == "attention":
                mixer = self._attention_dict(m)
            else:
                mixer = {"left": self._attention_dict(m["left"]), "right": {"width": m["right_width"]},
                         "left_scale": m["left_scale"], "right_scale": m["right_scale"]}
            mlp = None
            if layer.mlp is not None:
                f = layer.mlp
                mlp = {"kind": "moe", "expert": {"ff": f["ff"]}, "router": {"experts": f["experts"], "top": f["top"]},
                       "shared": None if f["shared_ff"] is None else {"ff": f["shared_ff"]}}
            out_layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.ARCHITECTURE, "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
                             "residual_mult": self.residual_mult, "layers": out_layers}
        if self.bigram is not None:
            d["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), self.bigram))}
        if self.loop is not None:
            d["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- the model this configuration describes ----------------------------------------------------
    def run_plan(self) -> List[int]:
        """Layer numbers in execution order."""
        n = len(self.layers)
        start, stop, times = self.loop if self.loop is not None else (0, 0, 1)
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    def to_spec(self) -> ModelSpec:
        rotations: Dict[Tuple, str] = {}

        def rotation(dims: int, base: float, scaling: Optional[Tuple] = None) -> str:
            return rotations.setdefault((dims, base, scaling), f"rot{len(rotations)}")

        def common(m) -> Dict[str, Any]:
            return {"hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                    "value_dim": m["vdim"], "scale": m["scale"], "eps": self.eps, "softcap": m["softcap"], "window": m["window"],
                    "pairs": "halves", "position": rotation(m["rot_dims"], m["rot_base"], m["rot_scaling"])}

        norm = PartSpec("rmsnorm", {"size": self.width, "eps": self.eps, "tensor": ""}, "norm")
        specs = []
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if layer.type == "attention":
                mixer = PartSpec("differential_attention", {**common(m), "diff": m["diff"], "bias": True}, "mixer")
            else:
                left = {**common(m["left"]), "gate": False, "slot_multiple": 16,
                        "value_position": rotation(m["left"]["vdim"], m["left"]["rot_base"])}
                mixer = PartSpec("parallel_mixers", {"branches": [
                    {"kind": "unit_qk_attention", "params": left, "prefix": "left.", "scale": m["left_scale"]},
                    {"kind": "min_gru", "params": {"hidden_size": self.width, "width": m["right_width"]}, "prefix": "right.",
                     "scale": m["right_scale"]}]}, "mixer")
            parts = {"mixer": mixer, "mixer_norm": norm}
            names = {"mixer": "mix.", "mixer_norm": "norm1"}
            if layer.mlp is not None:
                f = layer.mlp
                parts["feed_forward"] = PartSpec("routed_moe", {
                    "hidden_size": self.width, "intermediate_size": f["ff"], "experts": f["experts"], "top": f["top"],
                    "shared_intermediate_size": f["shared_ff"], "activation": "silu", "scoring": "softmax", "weight_eps": 0.0,
                    "correction": "router.b"}, "feed_forward")
                parts["feed_forward_norm"] = norm
                names.update({"feed_forward": "mlp.", "feed_forward_norm": "norm2"})
            specs.append(LayerSpec(f"l{i}.", PartSpec("side_by_side_residual", {"multiplier": self.residual_mult}), parts, names))
        hooks = ()
        if self.bigram is not None:
            buckets, mul_prev, mul_cur = self.bigram
            hooks = (PartSpec("bigram_rows", {"width": self.width, "buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur,
                                              "tensor": "bigram"}),)
        encodings = {key: PartSpec("rotary", {
            "head_dim": dims, "theta": base, "rotary_dim": dims,
            "scaling": None if scaling is None else dict(zip(SCALING, scaling), rope_type="yarn")})
            for (dims, base, scaling), key in rotations.items()}
        return ModelSpec(
            architecture=self.ARCHITECTURE, hidden_size=self.width, vocab_size=self.vocab,
            max_position_embeddings=self.max_positions, embedding_name="embed", layers=tuple(specs),
            # every pass over a layer has a cache (and state) of its own
            run_order=tuple(RunEntry(layer=i, cache=n) for n, i in enumerate(self.run_plan())),
            final_norm=PartSpec("rmsnorm", {"size": self.width, "eps": self.eps, "tensor": ""}), final_norm_prefix="final.norm",
            lm_head_name="head", position_encodings=encodings, embedding_hooks=hooks, residual_dtype="float32",
            eos_token_ids=self.eos_token_ids,
            # the kernels of this design are those on which programmatic dependent launch is not trusted (see `TugodraConfig`)
            programmatic_launch=False)

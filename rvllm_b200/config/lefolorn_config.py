"""Configuration of the Lefolorn decoder: layers listed one by one.  A layer has ONE norm (an RMSNorm in groups); its mixer and
its feed-forward stand side by side and both read the norm's output, and what each returns is multiplied element by element by a
learned vector and by a sigmoid of a projection of that same output before it joins the float32 stream.  A mixer is grouped-query
attention without positions but with a learned bias per distance, window attention on turned queries and keys with capped
scores, or latent attention with a sink; the first two norm queries and keys per head and may mix the first such layer's
values into their own.  The feed-forward is a routed mixture of gated experts, some of which may be the identity.

config.json keys (all sizes and every constant that may differ between models are read, none is assumed):

    architecture            "Lefolorn"
    width, vocab            model width and vocabulary size
    norm.eps, norm.groups   eps of every norm; into how many equal parts the model's norms split a row
    layers[i].type          "attention" | "attention_2" | "latent_attention"
    layers[i].mixer         attention: heads, kv_heads, dim, vdim, scale, bias_max, q_temp.{coef, every} (absent: none),
                                       v_mix (absent: false), bias_rows (optional: rows of the distance table where weights are
                                       drawn at random; a checkpoint's own number counts)
                            attention_2: heads, kv_heads, dim, vdim, scale, rot.{dims, base}, softcap (absent: no cap),
                                       mask.size (absent: every earlier key), v_mix (absent: false)
                            latent_attention: heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot.{dims, base}
    layers[i].mlp           null | {"kind": "moe", "expert": {"ff": n}, "router": {"experts": E, "top": k,
                                    "identity": I (absent: 0), "groups": {"count": c, "keep": m} (absent: one group)},
                                    "shared": {"ff": m} | null}
    max_positions           optional: the longest sequence the rotation tables are ever built for

Tensor names: embed, head, final.norm, l<i>.{norm1, ls1, ls2, rg1, rg1.b, rg2, rg2.b}, l<i>.mix.{q, q.b, k, k.b, v, v.b, q.norm,
k.norm, vmix, o} (attention: and rel, g) | l<i>.mix.{dq, dq.norm, uq, dkv, dkv.norm, uk, uv, sink, o},
l<i>.mlp.{router, correction, e<j>.gate, e<j>.up, e<j>.down, shared.gate, shared.up, shared.down}.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from ..errors import ConfigError
from .reader import NumberReader, is_int
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

DEFAULT_MAX_POSITIONS = 1 << 17       # the design sets no limit; the engine's tables are built for max_model_len
DEFAULT_BIAS_ROWS = 32                # rows of a distance table drawn at random
MIXERS = ("attention", "attention_2", "latent_attention")


@dataclass(frozen=True)
class LefolornLayer:
    type: str                              # one of MIXERS
    mixer: Dict[str, Any]                  # the mixer's sizes and constants, flat (rot_dims, rot_base, window, temp_coef, ...)
    mlp: Optional[Dict[str, Any]]          # None | {ff, experts, identity, top, groups, keep, shared_ff | None}


class _Reader(NumberReader):
    def rotation(self, m, at: str, inside: int, what: str) -> Tuple[int, float]:
        rot = m.get("rot")
        dims = self.integer(rot, "dims", at + "rot: ", minimum=2)
        base = self.number(rot, "base", at + "rot: ")
        if dims % 2 or dims > inside:
            self.problems.append(at + f"`rot.dims` must be even and at most {what} = {inside}, got {dims}")
        return dims, base

    def mixer(self, kind: str, m, at: str) -> Dict[str, Any]:
        if not isinstance(m, dict):
            self.problems.append(at + "`mixer` must be an object")
            m = {}
        if kind == "latent_attention":
            out: Dict[str, Any] = {key: self.integer(m, key, at) for key in ("heads", "dim", "vdim", "q_rank", "kv_rank")}
            out["rot_dim"] = self.integer(m, "rot_dim", at, minimum=2)
            out["scale"] = self.number(m, "scale", at)
            out["rot_dims"], out["rot_base"] = self.rotation(m, at, out["rot_dim"], "rot_dim")
            return out
        out = {key: self.integer(m, key, at) for key in ("heads", "kv_heads", "dim", "vdim")}
        out["scale"] = self.number(m, "scale", at)
        if out["heads"] % out["kv_heads"]:
            self.problems.append(at + f"{out['heads']} query heads cannot share {out['kv_heads']} key/value heads")
        out["v_mix"] = m.get("v_mix", False)
        if not isinstance(out["v_mix"], bool):
            self.problems.append(at + f"`v_mix` must be true or false, got {out['v_mix']!r}")
        if kind == "attention":
            out["bias_max"] = self.number(m, "bias_max", at)
            out["bias_rows"] = self.integer(m, "bias_rows", at, minimum=2) if "bias_rows" in m else DEFAULT_BIAS_ROWS
            temp = m.get("q_temp")
            out["temp_coef"] = None if temp is None else self.number(temp, "coef", at + "q_temp: ", positive=False)
            if isinstance(temp, dict) and isinstance(temp.get("every"), float) and temp["every"].is_integer():
                temp = dict(temp, every=int(temp["every"]))
            out["temp_every"] = None if temp is None else self.integer(temp, "every", at + "q_temp: ")
        else:
            out["rot_dims"], out["rot_base"] = self.rotation(m, at, out["dim"], "dim")
            cap, mask = m.get("softcap"), m.get("mask")
            out["softcap"] = None if cap is None else self.number(m, "softcap", at)
            out["window"] = None if mask is None else self.integer(mask, "size", at + "mask: ")
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
               "top": self.integer(router, "top", at + "mlp.router: "), "identity": 0, "groups": 1, "keep": 1, "shared_ff": None}
        router = router if isinstance(router, dict) else {}
        if router.get("identity") is not None:
            mlp["identity"] = self.integer(router, "identity", at + "mlp.router: ", minimum=0)
        groups = router.get("groups")
        if groups is not None:
            mlp["groups"] = self.integer(groups, "count", at + "mlp.router.groups: ")
            mlp["keep"] = self.integer(groups, "keep", at + "mlp.router.groups: ")
        total = mlp["experts"] + mlp["identity"]
        if total % mlp["groups"] or mlp["keep"] > mlp["groups"]:
            self.problems.append(at + f"mlp.router: {total} experts in {mlp['groups']} equal groups of which {mlp['keep']} are kept")
        elif mlp["top"] > mlp["keep"] * (total // mlp["groups"]):
            self.problems.append(at + f"mlp.router: `top` {mlp['top']} exceeds the experts of the {mlp['keep']} kept groups")
        if raw.get("shared") is not None:
            mlp["shared_ff"] = self.integer(raw.get("shared"), "ff", at + "mlp.shared: ")
        return mlp


@dataclass(frozen=True)
class LefolornConfig:
    width: int
    vocab: int
    eps: float
    norm_groups: int
    layers: Tuple[LefolornLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_ids: Tuple[int, ...] = ()
    raw: Dict[str, Any] = field(default_factory=dict, compare=False, repr=False)

    ARCHITECTURE = "Lefolorn"

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
    def from_dict(cls, obj: Dict[str, Any], where: str = "config.json") -> "LefolornConfig":
        r = _Reader()
        p = r.problems
        width = r.integer(obj, "width", "")
        vocab = r.integer(obj, "vocab", "")
        eps = r.number(obj.get("norm"), "eps", "norm: ")
        groups = r.integer(obj.get("norm"), "groups", "norm: ")
        if width % groups:
            p.append(f"norm: a width of {width} does not split into {groups} equal groups")
        raw_layers = obj.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError(p + ["`layers` must be a non-empty list"], where)
        layers: List[LefolornLayer] = []
        mixed_values: Optional[Tuple[int, int]] = None          # (layer, elements per token) of the first layer that mixes values
        for i, e in enumerate(raw_layers):
            at = f"layers[{i}]: "
            if not isinstance(e, dict):
                p.append(at + "must be an object")
                continue
            kind = e.get("type")
            if kind not in MIXERS:
                p.append(at + f"`type` = {kind!r} is not known ({', '.join(MIXERS)})")
                continue
            mixer = r.mixer(kind, e.get("mixer"), at)
            if mixer.get("v_mix"):
                size = mixer["kv_heads"] * mixer["vdim"]
                if mixed_values is None:
                    mixed_values = (i, size)
                elif mixed_values[1] != size:
                    p.append(at + f"`v_mix`: values of {size} elements cannot take a share of layer {mixed_values[0]}'s {mixed_values[1]}")
            layers.append(LefolornLayer(kind, mixer, r.moe(e.get("mlp"), at)))
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
        return cls(width=width, vocab=vocab, eps=eps, norm_groups=groups, layers=tuple(layers), max_positions=max_pos,
                   eos_token_ids=eos_ids, raw=dict(obj))

    # ---- writing -------------------------------------------------------------------------------
    def to_dict(self) -> Dict[str, Any]:
        out_layers = []
        for layer in self.layers:
            m = dict(layer.mixer)
            if "rot_dims" in m:
                m["rot"] = {"dims": m.pop("rot_dims"), "base": m.pop("rot_base")}
            if layer.type == "attention":
                coef, every = m.pop("temp_coef"), m.pop("temp_every")
                if coef is not None:
                    m["q_temp"] = {"coef": coef, "every": every}
                if m["bias_rows"] == DEFAULT_BIAS_ROWS:
                    del m["bias_rows"]
            elif layer.type == "attention_2":
                window = m.pop("window")
                if window is not None:
                    m["mask"] = {"size": window}
                if m["softcap"] is None:
                    del m["softcap"]
            mlp = None
            if layer.mlp is not None:
                f = layer.mlp
                mlp = {"kind": "moe", "expert": {"ff": f["ff"]},
                       "router": {"experts": f["experts"], "top": f["top"], "identity": f["identity"],
                                  "groups": {"count": f["groups"], "keep": f["keep"]}},
                       "shared": None if f["shared_ff"] is None else {"ff": f["shared_ff"]}}
            out_layers.append({"type": layer.type, "mixer": m, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.ARCHITECTURE, "width": self.width, "vocab": self.vocab,
                             "norm": {"eps": self.eps, "groups": self.norm_groups}, "layers": out_layers}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- the model this configuration describes ----------------------------------------------------
    def to_spec(self) -> ModelSpec:
        rotations: Dict[Tuple[int, float], str] = {}
        mixing = [i for i, layer in enumerate(self.layers) if layer.mixer.get("v_mix")]
        norm = PartSpec("grouped_rmsnorm", {"size": self.width, "groups": self.norm_groups, "eps": self.eps, "tensor": ""}, "norm")
        specs, ignored = [], []
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            position = None
            if "rot_dims" in m:
                position = rotations.setdefault((m["rot_dims"], m["rot_base"]), f"rot{len(rotations)}")
            if layer.type == "latent_attention":
                mixer = PartSpec("latent_attention", {
                    "hidden_size": self.width, "num_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"],
                    "value_dim": m["vdim"], "kv_rank": m["kv_rank"], "q_rank": m["q_rank"], "scale": m["scale"], "eps": self.eps,
                    "gate": False, "sink": True, "pairs": "neighbours", "position": position, "suffix": ""}, "mixer")
            else:
                params = {"hidden_size": self.width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                          "value_dim": m["vdim"], "scale": m["scale"], "eps": self.eps, "bias": True, "position": position,
                          "pairs": "neighbours", "value_mix": None if not m["v_mix"] else ("first" if i == mixing[0] else "later")}
                if layer.type == "attention":
                    params.update(distance_limit=m["bias_max"], distance_rows=m["bias_rows"], unit_sink=True, gate=True,
                                  temperature=None if m["temp_coef"] is None else (m["temp_coef"], m["temp_every"]))
                else:
                    params.update(softcap=m["softcap"], window=m["window"])
                mixer = PartSpec("normed_qk_attention", params, "mixer")
            parts = {"mixer": mixer, "norm": norm}
            names = {"mixer": "mix.", "norm": "norm1"}
            if layer.mlp is not None:
                f = layer.mlp
                parts["feed_forward"] = PartSpec("routed_moe", {
                    "hidden_size": self.width, "intermediate_size": f["ff"], "experts": f["experts"], "identity": f["identity"],
                    "top": f["top"], "groups": f["groups"], "keep_groups": f["keep"], "group_score": "max",
                    "shared_intermediate_size": f["shared_ff"], "shared_gate": None, "activation": "silu", "scoring": "softmax_all"},
                    "feed_forward")
                names["feed_forward"] = "mlp."
            else:                          # what would stand behind a feed-forward has nothing to act on
                ignored += [f"l{i}.ls2", f"l{i}.rg2", f"l{i}.rg2.b"]
            specs.append(LayerSpec(f"l{i}.", PartSpec("shared_norm_gated_residual", {"hidden_size": self.width}), parts, names))
        return ModelSpec(
            architecture=self.ARCHITECTURE, hidden_size=self.width, vocab_size=self.vocab,
            max_position_embeddings=self.max_positions, embedding_name="embed", layers=tuple(specs),
            run_order=tuple(RunEntry(layer=i, cache=i) for i in range(len(specs))),
            final_norm=PartSpec("grouped_rmsnorm", dict(norm.params)), final_norm_prefix="final.norm", lm_head_name="head",
            ignored_tensors=tuple(ignored),
            position_encodings={key: PartSpec("rotary", {"head_dim": dims, "theta": base, "rotary_dim": dims})
                                for (dims, base), key in rotations.items()},
            residual_dtype="float32", eos_token_ids=self.eos_token_ids,
            # the kernels of this design are those on which programmatic dependent launch is not trusted (see `TugodraConfig`)
            programmatic_launch=False)

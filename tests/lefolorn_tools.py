"""Small Lefolorn configurations, model folders for them and plain logits, for the tests of that design.

The sizes differ from layer to layer and between the configurations and avoid values that hide a fault: value sizes unlike key
sizes (smaller and larger), rotations of part of a head, head groups of one and of several, windows that divide neither a page
nor a tile and none at all, scores with and without a cap, distance tables with even and odd and very few rows, query
temperatures that grow often, seldom and not at all, the first layer that mixes values at different places and of either kind,
routers with and without groups, identity experts and a shared expert, one choice and all of them, a layer without a
feed-forward, one norm group and one of four columns."""
from __future__ import annotations

import copy
from typing import Dict, List, Optional

import torch

import plain_lefolorn as P
from tufirax_tools import read_folder, write_folder      # (folders are written by the framework's random-weights mode)


def moe(ff=24, experts=6, top=2, identity=0, groups: Optional[tuple] = None, shared: Optional[int] = 16):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router, "shared": None if shared is None else {"ff": shared}}


def attention(heads=4, kv_heads=2, dim=24, vdim=16, rows=12, bias_max=40, temp: Optional[tuple] = (0.7, 5), scale=0.25, v_mix=False, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max, "bias_rows": rows, "v_mix": v_mix}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": copy.deepcopy(mlp)}


def window(heads=6, kv_heads=2, dim=12, vdim=20, size: Optional[int] = 13, rot_dims=8, base=500.0, scale=0.4, softcap: Optional[float] = 9.0,
           v_mix=False, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot_dims, "base": base}, "v_mix": v_mix}
    if size is not None:
        m["mask"] = {"size": size}
    if softcap is not None:
        m["softcap"] = softcap
    return {"type": "attention_2", "mixer": m, "mlp": copy.deepcopy(mlp)}


def latent(heads=5, dim=14, rot_dim=6, vdim=10, q_rank=18, kv_rank=22, base=300.0, scale=0.3, mlp=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"dims": rot_dim, "base": base}}, "mlp": copy.deepcopy(mlp)}


def config(layers: List[dict], width=48, vocab=131, eps=1e-5, groups=3) -> dict:
    return {"architecture": "Lefolorn", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups}, "layers": copy.deepcopy(layers)}


def small_a() -> dict:
    """All mixers in unlike sizes; the second layer is the first that mixes values."""
    return config([window(mlp=moe(identity=2, groups=(4, 2), top=3)),
                   attention(v_mix=True, mlp=moe(ff=20, experts=5, top=1, shared=None)),
                   latent(mlp=moe(ff=16, experts=3, identity=1, top=4, shared=24)),
                   window(heads=2, kv_heads=2, dim=16, vdim=16, size=7, rot_dims=16, base=40.0, scale=0.6, softcap=None, v_mix=True),
                   latent(heads=3, dim=8, rot_dim=10, vdim=12, q_rank=9, kv_rank=17, base=20.0, scale=0.5, mlp=moe(experts=7, top=7, shared=8)),
                   attention(heads=6, kv_heads=2, dim=10, vdim=16, rows=5, bias_max=9, temp=None, scale=0.7, v_mix=True,
                             mlp=moe(experts=4, identity=5, top=2, groups=(3, 1), shared=20))])


def small_b() -> dict:
    """Sizes the tensor-core kernels are built for: heads of 64, 80 and 128, a latent row of 128, groups of four, multiples of
    16 everywhere, a window and a distance table that end inside a page and inside a 64-key tile."""
    return config([attention(heads=8, kv_heads=2, dim=64, vdim=64, rows=32, bias_max=100, temp=(0.3, 32), scale=0.125, v_mix=True,
                             mlp=moe(ff=32, experts=6, identity=2, top=3, groups=(4, 3), shared=48)),
                   window(heads=8, kv_heads=2, dim=80, vdim=64, size=75, rot_dims=32, base=1e5, scale=0.11, softcap=15.0, v_mix=True,
                          mlp=moe(ff=48, experts=4, top=2, shared=32)),
                   latent(heads=4, dim=32, rot_dim=32, vdim=48, q_rank=40, kv_rank=96, base=1e4, scale=0.125, mlp=moe(ff=16, experts=4, identity=2, top=2)),
                   window(heads=4, kv_heads=1, dim=128, vdim=128, size=40, rot_dims=64, base=1e6, scale=0.09, softcap=30.0, v_mix=True)],
                  width=512, vocab=203, eps=1e-6, groups=2)


def odd_shapes() -> dict:
    """Sizes that no fast path is made for: a width and a vocabulary that are no multiples of 8, odd key, value and latent sizes,
    one head, a window of one key and none, distance tables of two and three rows, norm groups of four columns.  Its routers have few
    close calls, which rounding would decide either way."""
    return config([attention(heads=3, kv_heads=3, dim=9, vdim=7, rows=2, bias_max=3, temp=(1.5, 1), v_mix=True,
                             mlp=moe(ff=9, experts=1, identity=3, top=2, groups=(2, 1), shared=5)),
                   window(heads=1, kv_heads=1, dim=10, vdim=14, size=1, rot_dims=6, base=7.0, mlp=moe(ff=11, experts=1, top=1, shared=None)),
                   latent(heads=1, dim=3, rot_dim=2, vdim=5, q_rank=7, kv_rank=9, base=3.0, mlp=moe(ff=7, experts=9, top=9, shared=13)),
                   attention(heads=3, kv_heads=1, dim=5, vdim=21, rows=3, bias_max=60, temp=(-0.2, 64), v_mix=False),
                   window(heads=6, kv_heads=3, dim=33, vdim=7, size=None, rot_dims=2, base=11.0, softcap=4.0, v_mix=True, mlp=moe(identity=1, experts=2, top=3, shared=3))],
                  width=44, vocab=77, groups=11)


def lively(tensors: Dict[str, torch.Tensor], seed: int = 1) -> None:
    """Make the random weights show more: larger matrices inside the mixers (scores that reach the caps), distance biases and
    sinks that matter, routers that decide clearly with corrections that change the choice, gates over their whole range,
    weights of the norms and vectors that differ."""
    g = torch.Generator().manual_seed(seed)
    for name in sorted(tensors):
        t = tensors[name]

        def fill(lo, hi):
            t.copy_((torch.rand(t.shape, generator=g) * (hi - lo) + lo).to(t.dtype))
        if name == "embed":
            t.mul_(30.0)
        elif name.endswith((".q.b", ".k.b", ".v.b")):
            fill(-0.8, 0.8)
        elif name.endswith((".q.norm", ".k.norm", ".dq.norm", ".dkv.norm")):
            fill(0.4, 1.8)
        elif name.endswith(".mix.rel"):
            fill(-2.0, 2.5)
        elif name.endswith(".mix.sink"):
            fill(-2.0, 3.0)
        elif name.endswith(".mix.vmix"):
            fill(0.3, 0.8)
        elif ".mix." in name:
            t.mul_(9.0)
        elif name.endswith(".mlp.router"):
            t.mul_(15.0)
        elif name.endswith(".mlp.correction"):
            fill(-0.3, 0.3)
        elif ".mlp." in name:
            t.mul_(8.0)
        elif name.endswith((".rg1.b", ".rg2.b")):
            fill(-1.0, 2.0)
        elif name.endswith((".rg1", ".rg2")):
            t.mul_(10.0)
        elif name.endswith(("norm1", "final.norm", ".ls1", ".ls2")):
            fill(0.4, 1.6)
        elif name == "head":
            t.mul_(5.0)


def plain_logits(folder: str, requests: Dict[str, List[int]], rounded: bool = False) -> Dict[str, torch.Tensor]:
    cfg, w = read_folder(folder)
    store = P.round_to_bfloat16 if rounded else P._keep
    return {rid: P.forward(cfg, w, toks, store=store) for rid, toks in requests.items()}

"""Small Sozudra configurations, model folders for them and plain logits, for the tests of that design.

The sizes differ from layer to layer and between the configurations and avoid values that hide a fault: value sizes
unlike key sizes (smaller and larger, and unlike two maps of a key), rotations of part of a head with and without a scaling
of their frequencies, head groups of one and of several, windows that divide neither a page nor a tile and none at all,
scores with and without a cap, looped spans at the start, in the middle and none, routers that choose one expert and all of
them, experts without a shared one, layers without a feed-forward, a model without bigram rows."""
from __future__ import annotations

import copy
from typing import Dict, List, Optional

import torch

import plain_sozudra as P
from tufirax_tools import read_folder, write_folder      # (folders are written by the framework's random-weights mode)

YARN = {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 1.5}


def moe(ff=24, experts=6, top=2, shared: Optional[int] = 16):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top},
            "shared": None if shared is None else {"ff": shared}}


def _heads(heads, kv_heads, dim, vdim, window, rot_dims, base, scaling, scale, softcap):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot_dims or dim, "base": base}}
    if window is not None:
        m["mask"] = {"size": window}
    if scaling is not None:
        m["rot"]["scaling"] = dict(scaling)
    if softcap is not None:
        m["softcap"] = softcap
    return m


def attention(heads=6, kv_heads=2, dim=12, vdim=20, window: Optional[int] = 13, rot_dims=None, base=500.0, scaling=YARN, scale=0.4,
              softcap: Optional[float] = 9.0, diff=0.35, mlp=None):
    return {"type": "attention", "mixer": dict(_heads(heads, kv_heads, dim, vdim, window, rot_dims, base, scaling, scale, softcap), diff=diff),
            "mlp": copy.deepcopy(mlp)}


def parallel(heads=4, kv_heads=2, dim=24, vdim=16, window: Optional[int] = 11, rot_dims=None, base=300.0, scaling=YARN, scale=0.3,
             softcap: Optional[float] = 6.0, width=40, left_scale=0.7, right_scale=1.3, mlp=None):
    return {"type": "parallel", "mixer": {"left": _heads(heads, kv_heads, dim, vdim, window, rot_dims, base, scaling, scale, softcap),
                                          "right": {"width": width}, "left_scale": left_scale, "right_scale": right_scale},
            "mlp": copy.deepcopy(mlp)}


def config(layers: List[dict], width=48, vocab=131, eps=1e-5, mult=0.6, bigram=(37, 5, 11), loop=None) -> dict:
    d = {"architecture": "Sozudra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
         "layers": copy.deepcopy(layers)}
    if bigram is not None:
        d["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


def small_a() -> dict:
    """Both mixers in unlike sizes; a span in the middle runs three times; values narrower and wider than keys, part of a
    head rotated, one expert of several and all of them, no cap, no window, no scaling, no shared expert, no feed-forward."""
    return config([attention(mlp=moe()),
                   parallel(mlp=moe(ff=20, experts=5, top=1, shared=None)),
                   attention(heads=4, kv_heads=4, dim=8, vdim=12, window=29, rot_dims=4, base=30.0, scaling=None, scale=0.5, softcap=None,
                             diff=0.1, mlp=moe(ff=16, experts=3, top=3, shared=24)),
                   parallel(heads=6, kv_heads=1, dim=8, vdim=20, window=None, rot_dims=6, base=40.0, scaling=None, scale=0.6, softcap=None,
                            width=33, left_scale=1.2, right_scale=-0.5, mlp=None),
                   attention(heads=2, kv_heads=1, dim=16, vdim=36, window=7, base=2000.0, softcap=3.0, diff=0.8, mlp=None)],
                  loop=(1, 3, 3))


def small_b() -> dict:
    """Sizes the tensor-core kernels are built for: heads of 64 and two maps of 32 with values of 64, groups of four, multiples
    of 16 everywhere, windows that end inside a page and inside a 64-key tile; the loop starts at the first layer."""
    return config([parallel(heads=8, kv_heads=2, dim=64, vdim=64, window=75, base=1e5, scale=0.125, softcap=15.0, width=96,
                            scaling={"factor": 8.0, "original": 256, "fast": 32.0, "slow": 1.0},
                            mlp=moe(ff=32, experts=8, top=3, shared=48)),
                   attention(heads=8, kv_heads=2, dim=32, vdim=64, window=40, rot_dims=16, base=1e6, scale=0.18, softcap=30.0, diff=0.25,
                             scaling={"factor": 2.0, "original": 128, "fast": 8.0, "slow": 2.0}, mlp=moe(ff=48, experts=4, top=2, shared=32))],
                  width=64, vocab=203, eps=1e-6, mult=0.8, bigram=(97, 1009, 3), loop=(0, 2, 2))


def odd_shapes() -> dict:
    """Sizes that no fast path is made for: a width and a vocabulary that are no multiples of 8, odd key sizes, one head, a
    window of one key and one of five, no bigram rows, no loop."""
    return config([parallel(heads=3, kv_heads=3, dim=10, vdim=14, window=5, rot_dims=6, base=7.0, width=37, mlp=moe(ff=9, experts=4, top=2, shared=5)),
                   attention(heads=1, kv_heads=1, dim=9, vdim=7, window=1, rot_dims=4, base=3.0, mlp=moe(ff=11, experts=1, top=1, shared=None)),
                   attention(heads=6, kv_heads=3, dim=5, vdim=33, window=33, rot_dims=2, base=11.0, softcap=None, mlp=None),
                   parallel(heads=5, kv_heads=5, dim=21, vdim=6, window=18, rot_dims=20, base=60.0, width=130, mlp=moe(ff=7, experts=9, top=4, shared=13))],
                  width=44, vocab=77, mult=1.1, bigram=None)


def lively(tensors: Dict[str, torch.Tensor], seed: int = 1) -> None:
    """Make the random weights show more: larger matrices inside the mixers (scores that reach the caps), gates of the
    recurrence between fast and slow, candidates of both signs, routers that decide clearly with biases that change the
    choice, norm weights that differ, a bigram row as large as a token's."""
    g = torch.Generator().manual_seed(seed)
    for name in sorted(tensors):
        t = tensors[name]

        def fill(lo, hi):
            t.copy_((torch.rand(t.shape, generator=g) * (hi - lo) + lo).to(t.dtype))
        if name in ("embed", "bigram"):
            t.mul_(30.0)
        elif name.endswith((".q.b", ".k.b", ".v.b")):
            fill(-0.8, 0.8)
        elif ".mix." in name and name.endswith((".q", ".k")):
            t.mul_(12.0)
        elif ".mix." in name and name.endswith((".v", ".o", ".g")):
            t.mul_(7.0)
        elif name.endswith((".right.z", ".right.x")):
            t.mul_(15.0)
        elif name.endswith(".right.z.b"):
            fill(-4.0, 2.0)
        elif name.endswith(".right.x.b"):
            fill(-1.5, 1.5)
        elif name.endswith(".mlp.router"):
            t.mul_(20.0)
        elif name.endswith(".mlp.router.b"):
            fill(-0.7, 0.7)
        elif name.endswith(".mlp.shared.sg"):
            t.mul_(20.0)
        elif ".mlp." in name:
            t.mul_(8.0)
        elif name.endswith(("norm1", "norm2", "final.norm")):
            fill(0.5, 1.8)
        elif name == "head":
            t.mul_(5.0)


def plain_logits(folder: str, requests: Dict[str, List[int]], rounded: bool = False) -> Dict[str, torch.Tensor]:
    cfg, w = read_folder(folder)
    store = P.round_to_bfloat16 if rounded else P._keep
    return {rid: P.forward(cfg, w, toks, store=store) for rid, toks in requests.items()}

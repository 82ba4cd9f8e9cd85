"""Tiny Saropel configurations and model folders shared by the tests.

Three configurations that differ from each other in every size and option:
  SA: width 64, vocab 200, a pair table of 53 buckets, 12 columns of token input (no multiple of 8), layers 1 and 2
      looped three times; capped attention with grouped heads (4 on 2), values wider than keys, a window of 9, 6 experts
      in 3 groups of which 2, top 3, and a shared expert with a limit of its own; shared-key attention under a window of
      20 with half of a head rotated by stretched frequencies and a dense feed-forward; capped attention under a window
      of ONE key without feed-forward; shared-key attention without grouping, mask or stretch, one of 4 experts, no shared
      expert, no groups
  SB: width 96, vocab 320, no pair table, no loop, 32 columns of token input; 20 query heads on one key/value head of 64,
      40 experts in 5 groups, top 5; capped attention with heads of 64 under a window of 33; 5 heads of 8 with 6
      dimensions rotated; capped attention without a mask, heads of 128, experts in groups that are all kept
  SC: width 36 (no multiple of 8), vocab 96, a pair table, no token input, both layers looped twice; 1 bucket is never
      enough to tell pairs apart, so there are 7; both of 2 experts chosen
"""
from __future__ import annotations

import math
from pathlib import Path

import torch


def rotation(base, dims, factor=None, original=64, fast=32.0, slow=1.0):
    r = {"base": base, "dims": dims}
    if factor:
        r["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return r


def capped(heads, kv_heads, dim, vdim, window, softcap, scale=0.3):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": softcap}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m}


def shared_kv(heads, kv_heads, dim, window, rot, scale=0.3):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if rot:
        m["rot"] = rot
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention_2", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=1.0, groups=None, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def bigram(buckets, mul_prev, mul_cur):
    return {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}


CONFIG_SA = {"architecture": "Saropel", "norm": {"eps": 1e-5}, "vocab": 200, "width": 64, "embedding": bigram(53, 5, 11),
             "token_side": {"dim": 12}, "loop": {"start": 1, "stop": 3, "times": 3},
             "layers": [dict(capped(4, 2, 16, 24, 9, 2.5), mlp=moe(6, 3, 24, 0.8, (3, 2), (40, 0.5))),
                        dict(shared_kv(4, 2, 32, 20, rotation(1e3, 16, 3.0)), mlp=dense(48)),
                        dict(capped(2, 1, 16, 16, 1, 6.0), mlp=None),
                        dict(shared_kv(3, 3, 24, 0, rotation(1e4, 24)), mlp=moe(4, 1, 32, 1.5))]}
CONFIG_SB = {"architecture": "Saropel", "norm": {"eps": 1e-6}, "vocab": 320, "width": 96, "token_side": {"dim": 32},
             "layers": [dict(shared_kv(20, 1, 64, 70, rotation(1e4, 64, 8.0, 32, 4.0, 0.5), 0.2),
                             mlp=moe(40, 5, 16, 2.0, (5, 2), (16, 1.0))),
                        dict(capped(3, 3, 64, 64, 33, 3.0, 0.15), mlp=dense(80)),
                        dict(shared_kv(5, 5, 8, 12, rotation(100.0, 6, 2.0)), mlp=None),
                        dict(capped(2, 1, 128, 128, 0, 20.0, 0.1), mlp=moe(6, 4, 24, 0.7, (2, 2), (24, 0.6)))]}
CONFIG_SC = {"architecture": "Saropel", "norm": {"eps": 1e-5}, "vocab": 96, "width": 36, "embedding": bigram(7, 3, 2),
             "loop": {"start": 0, "stop": 2, "times": 2},
             "layers": [dict(capped(2, 1, 8, 8, 5, 1.0), mlp=dense(40)),
                        dict(shared_kv(2, 1, 12, 17, rotation(1e3, 4, 4.0)), mlp=moe(2, 2, 16, 1.0, None, (8, 2.0)))]}
CONFIGS = {"SA": CONFIG_SA, "SB": CONFIG_SB, "SC": CONFIG_SC}


def read_tensors(folder) -> dict:
    from flambeau_b200.weights.safetensors_io import SafetensorsFile
    f = SafetensorsFile(Path(folder) / "model.safetensors")
    tensors = {n: f.tensor(n).clone() for n in f.names()}
    f.close()
    return tensors


def write_tensors(folder, tensors: dict) -> None:
    from flambeau_b200.weights.safetensors_io import write_safetensors
    write_safetensors(Path(folder) / "model.safetensors", tensors)


def make_folder(folder, cfg: dict, seed: int, dtype: str, sharp: float = 0.25, steady_router: bool = False) -> Path:
    """A model folder with seeded random weights.  The maps that form queries and keys are redrawn with standard
    deviation `sharp`, so that scores spread over several units (beyond the caps) and a wrong, missing or extra key
    shows in the logits; the experts' first maps wide enough that the limits cut; what the sublayers write wide enough to
    matter beside the token input.  `steady_router` (for runs in bfloat16, where the rounding of a close call would
    send a token to another expert than the oracle's; the float32 runs route by the token): channel 0 of the stream is
    made the same positive number for every token, which no sublayer writes to (constant columns of both embedding tables,
    rows of zeros in every output map, no token input and no vector of a pass there), and every router reads that
    channel alone with a different factor per expert: the order of the experts is then the same for every token."""
    from flambeau_b200.config.saropel import SaropelConfig
    from flambeau_b200.weights.random_init import write_random_model
    folder = Path(folder)
    write_random_model(folder, SaropelConfig.from_dict(cfg), seed=seed, dtype=dtype)
    tensors = read_tensors(folder)
    g = torch.Generator().manual_seed(seed * 7919 + 13)
    spread = [((".mix.q", ".mix.k"), sharp), ((".mix.v", ".mix.g", ".side.gate"), 0.1), ((".mix.o", ".down"), 0.12),
              ((".gate", ".up"), 0.2), ((".router",), 0.5), (("embed", "bigram"), 0.3), (("loop.step",), 0.3)]
    for n in sorted(tensors):
        t = tensors[n]
        std = next((s for ends, s in spread if n.endswith(ends) and n != "side.embed"), None)
        if std is not None:
            t = tensors[n] = (torch.randn(t.shape, generator=g) * std).to(t.dtype)
        if not steady_router:
            continue
        if n == "embed":
            t[:, 0] = 0.4
        elif n == "bigram":
            t[:, 0] = 0.25
        elif n == "loop.step":
            t[:, 0] = 0.0
        elif n.endswith((".mix.o", ".down", ".side.proj")):
            t[0] = 0.0
        elif n.endswith(".norm1"):
            tensors[n] = t.clamp(min=-0.5)
        elif n.endswith(".router"):
            # (a power of two as the unit keeps the factors exact in bfloat16; the largest logit, factor x the
            # channel's value of at most about sqrt(width), stays where the softmax still tells the scores apart)
            unit = 2.0 ** math.floor(math.log2(8.0 / math.sqrt(t.shape[1]) / t.shape[0]))
            factors = (torch.randperm(t.shape[0], generator=g).float() + 1.0) * unit
            tensors[n] = torch.zeros_like(t)
            tensors[n][:, 0] = factors.to(t.dtype)
    write_tensors(folder, tensors)
    return folder

"""Tiny Sisadra configurations and model folders shared by the tests.

Three configurations that differ from each other in every size and option:
  DA: width 64, vocab 200, a scaled embedding with a pair table of 53 buckets; differential attention with grouped heads
      (4 on 2), values wider than keys, a quarter of a map rotated, chunks of 20 (no multiple of a page); latent attention;
      the recurrence with grouped heads (6 on 2), values narrower than keys, 4 taps, no feed-forward; chunks of ONE key
      without rotation; a recurrence with one tap and equal heads in front of a feed-forward
  DB: width 96, vocab 320, no pair table, no cap on the logits; 18 query heads on one key/value head (more than a tile of
      rows), maps of 16 in chunks of 48 (whole pages); 18 heads on latents of 80 without feed-forward; a recurrence with
      keys of 40 and values of 72, 2 taps; attention without chunks, maps of 32, values of 64, unscaled waves
  DC: width 36 (no multiple of 8), vocab 90, odd head sizes everywhere, chunks of 7, latents of 20, 3 taps
"""
from __future__ import annotations

from pathlib import Path

import torch


def rotation(base, dims, factor=None, low=1.0, high=4.0, original=64):
    r = {"base": base, "dims": dims}
    if factor:
        r["scaling"] = {"factor": factor, "low": low, "high": high, "original": original}
    return r


def attention(heads, kv_heads, dim, vdim, chunk, rot=None, scale=0.3, diff=0.4):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = rot
    return {"type": "attention", "mixer": m}


def latent(heads, dim, vdim, kv_rank, scale=0.3):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def bigram(buckets, mul_prev, mul_cur):
    return {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}


CONFIG_DA = {"architecture": "Sisadra", "norm": {"eps": 1e-5}, "vocab": 200, "width": 64, "logit_softcap": 12.0,
             "embedding": {"scale": 2.5, "bigram": bigram(53, 5, 11)},
             "layers": [dict(attention(4, 2, 32, 48, 20, rotation(1e4, 8, 3.0)), mlp=dense(80)),
                        dict(latent(3, 16, 24, 48), mlp=dense(40)),
                        dict(delta(6, 2, 24, 16, 4), mlp=None),
                        dict(attention(2, 1, 16, 16, 1), mlp=None),
                        dict(delta(3, 3, 16, 32, 1), mlp=dense(56))]}
CONFIG_DB = {"architecture": "Sisadra", "norm": {"eps": 1e-6}, "vocab": 320, "width": 96, "embedding": {"scale": 1.0},
             "layers": [dict(attention(18, 1, 16, 32, 48, rotation(500.0, 16, 4.0, 0.5, 2.0, 200), 0.25, 0.2), mlp=dense(64)),
                        dict(latent(18, 8, 16, 80, 0.35), mlp=None),
                        dict(delta(4, 2, 40, 72, 2), mlp=dense(104)),
                        dict(attention(4, 4, 32, 64, 0, rotation(1e4, 32), 0.2, 0.6), mlp=None)]}
CONFIG_DC = {"architecture": "Sisadra", "norm": {"eps": 1e-5}, "vocab": 90, "width": 36, "logit_softcap": 5.0,
             "embedding": {"scale": 0.5, "bigram": bigram(7, 3, 2)},
             "layers": [dict(delta(3, 1, 10, 6, 3), mlp=dense(20)),
                        dict(attention(3, 1, 10, 18, 7, rotation(300.0, 6, 2.0, 1.0, 8.0, 30)), mlp=None),
                        dict(latent(2, 6, 10, 20), mlp=dense(44))]}
CONFIGS = {"DA": CONFIG_DA, "DB": CONFIG_DB, "DC": CONFIG_DC}


def read_tensors(folder) -> dict:
    from flambeau_b200.weights.safetensors_io import SafetensorsFile
    f = SafetensorsFile(Path(folder) / "model.safetensors")
    tensors = {n: f.tensor(n).clone() for n in f.names()}
    f.close()
    return tensors


def write_tensors(folder, tensors: dict) -> None:
    from flambeau_b200.weights.safetensors_io import write_safetensors
    write_safetensors(Path(folder) / "model.safetensors", tensors)


def rank_of(name: str, cfg: dict, seed: int) -> int:
    """How wide the narrow middle of a map is (no key of the configuration says so): it differs between layers and between
    a layer's two maps."""
    layer = int(name.split(".")[0][1:])
    return (5, 8, 12, 24, 66)[(layer + seed + (2 if ".g" in name else 0)) % 5]


def make_folder(folder, cfg: dict, seed: int, dtype: str, sharp: float = 0.25) -> Path:
    """A model folder with seeded random weights.  The maps that form queries and keys are redrawn with standard
    deviation `sharp` (and the norms of q and k with a spread), so that scores spread over several units and a wrong,
    missing or extra key shows in the logits; what the sublayers write wide enough to matter; biases that are not small;
    rates of decay from slow to fast; narrow middles of several widths."""
    from flambeau_b200.config.sisadra import SisadraConfig
    from flambeau_b200.weights.random_init import write_random_model
    folder = Path(folder)
    write_random_model(folder, SisadraConfig.from_dict(cfg), seed=seed, dtype=dtype)
    tensors = read_tensors(folder)
    g = torch.Generator().manual_seed(seed * 7919 + 13)
    for n in sorted(tensors):
        t, leaf = tensors[n], n.rsplit(".", 1)[-1]
        shape, std, centre = list(t.shape), None, 0.0
        if n.endswith((".q.norm", ".k.norm")):
            std, centre = 0.5, 1.5
        elif n.endswith((".q", ".k", ".dkv", ".uk")):
            std = sharp
        elif n.endswith((".v", ".uv", ".b")):
            std = 0.15 if n.count(".") == 2 else 0.3          # (a recurrence's own map 'b', and the biases)
        elif leaf in ("a1", "g1"):
            shape[0], std = rank_of(n, cfg, seed), 0.2
        elif leaf in ("a2", "g2"):
            shape[1], std = rank_of(n, cfg, seed), 0.3
        elif leaf == "A_log":
            std, centre = 1.0, -2.0
        elif n.endswith((".mix.o", ".down")):
            std = 0.12
        elif leaf == "up":
            std = 0.2
        elif leaf in ("embed", "bigram", "head"):             # (logits of a few units: a cap bends them)
            std = 0.3
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            std = 0.2
        if std is not None:
            tensors[n] = (torch.randn(shape, generator=g) * std + centre).to(t.dtype)
    write_tensors(folder, tensors)
    return folder

"""Tiny Tudulix configurations of the tests and helpers around them.

A has sizes no kernel likes (nothing a multiple of 8, keys and values of different sizes, a rotation over part of a head, three
query heads to a key/value head, windows of odd lengths and none, a shared expert of another width and limit than the routed
ones and a layer without one, a layer without feed-forward) and a loop of three passes in its middle.  B has sizes the fast
kernels take and a loop that starts with the first layer.  C makes things equal or 1 that the others keep apart (one head, keys
as long as values, a rotation over the whole head, a window of one token, one expert, one expert a token, all experts a token,
equal limits, scales of 1, a loop of one pass over all layers).  D has no loop.
"""
import copy
import json
import os

import torch

from prelude_b200.weights.random_init import random_tensors
from prelude_b200.weights.safetensors_io import write_safetensors


def moe(experts, top, ff, limit, shared=None):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def attention_mixer(heads, kv_heads, dim, vdim, scale, base, dims, window):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": dims, "base": base}}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def latent_mixer(heads, dim, rot_dim, vdim, rank, scale, base, window):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"dims": rot_dim, "base": base}}
    if window is not None:
        m["mask"] = {"size": window}
    return m


def attention(mlp, *args):
    return {"type": "attention", "mixer": attention_mixer(*args), "mlp": mlp}


def latent(mlp, *args):
    return {"type": "latent_attention", "mixer": latent_mixer(*args), "mlp": mlp}


def model(vocab, width, eps, embedding, logits, layers, loop=None):
    out = {"architecture": "Tudulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embedding},
           "logit_scale": logits, "layers": layers}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


TUDULIX_A = model(103, 44, 1e-5, 3.5, 1.7, [
    attention(moe(5, 2, 11, 0.9, (14, 0.6)), 6, 2, 10, 7, 0.4, 50.0, 6, 9),
    latent(moe(7, 3, 9, 0.7), 3, 10, 6, 7, 13, 0.4, 50.0, 13),
    attention(None, 3, 3, 9, 9, 0.5, 200.0, 4, 21),
    latent(moe(6, 1, 10, 1.4, (5, 2.0)), 5, 6, 4, 9, 11, 0.5, 30.0, None),
    latent(None, 2, 9, 2, 5, 13, 0.6, 20.0, 6),
], (1, 4, 3))

TUDULIX_B = model(211, 128, 1e-6, 8.0, 0.25, [
    latent(moe(8, 2, 64, 1.5, (128, 0.8)), 4, 32, 16, 32, 64, 0.25, 10000.0, 40),
    attention(moe(16, 4, 32, 0.8, (64, 1.2)), 4, 2, 64, 64, 0.2, 5000.0, 32, 24),
    attention(moe(4, 2, 96, 1.0), 8, 1, 32, 48, 0.25, 10000.0, 32, 70),
    latent(moe(12, 3, 48, 2.0, (64, 1.0)), 8, 16, 16, 64, 64, 0.25, 1000.0, 33),
], (0, 3, 2))

TUDULIX_C = model(50, 32, 1e-4, 1.0, 1.0, [
    attention(moe(1, 1, 8, 1.0, (8, 1.0)), 1, 1, 16, 16, 1.0, 20.0, 16, 1),
    latent(moe(3, 3, 16, 1.0), 1, 8, 8, 8, 8, 1.0, 20.0, 8),
    attention(moe(4, 1, 8, 1.0, (16, 1.0)), 4, 4, 8, 8, 1.0, 20.0, 2, 8),
], (0, 3, 1))

TUDULIX_D = model(97, 64, 1e-5, 2.0, 1.3, [
    attention(moe(6, 2, 24, 1.1, (40, 0.9)), 4, 4, 32, 32, 0.3, 100.0, 16, 17),
    latent(moe(6, 2, 24, 1.1, (40, 0.9)), 2, 16, 8, 16, 24, 0.35, 100.0, 30),
])

# configuration, random-weight options, page size
PARAMS = {"A": (TUDULIX_A, dict(seed=81, std=0.25, norm_jitter=0.3), 4),
          "B": (TUDULIX_B, dict(seed=82, std=0.12, norm_jitter=0.2), 16),
          "C": (TUDULIX_C, dict(seed=83, std=0.3, norm_jitter=0.2), 8),
          "D": (TUDULIX_D, dict(seed=84, std=0.2, norm_jitter=0.2), 8)}


def tensors_of(cfg: dict, dtype=None, decided=None, **init):
    """Random tensors; router logits are spread wide enough for clear choices, their biases of order one.  ``decided`` (in
    bfloat16 unless said otherwise): the biases lift as many experts as a token takes far above the others, so that no rounding
    of a router's input can turn a choice, which would change the logits outright; the weights still differ from token to
    token."""
    decided = dtype == torch.bfloat16 if decided is None else decided
    out = {}
    for k, v in random_tensors(cfg, **init).items():
        if k.endswith(".router"):
            v = v * 3.0
        elif k.endswith(".router.b"):
            v = v * 4.0
            if decided:
                top = cfg["layers"][int(k[1:k.index(".")])]["mlp"]["router"]["top"]
                v = v + 60.0 * (torch.randperm(v.numel(), generator=torch.Generator().manual_seed(len(k) + v.numel())) < top)
        out[k] = v if dtype is None else v.to(dtype)
    return out


def make_folder(tmp_path, which: str, dtype, config=None, **overrides):
    cfg, init, _ = PARAMS[which]
    cfg = copy.deepcopy(config or cfg)
    init = dict(init, **overrides)
    name = f"tudulix_{which}_{str(dtype).split('.')[-1]}_{abs(hash(str(cfg) + str(init))) % 10**8}"
    return make_folder_from_tensors(tmp_path, name, cfg, tensors_of(cfg, dtype, **init))


def make_folder_from_tensors(tmp_path, name: str, cfg: dict, tensors: dict) -> str:
    """A folder with the given tensors (made or changed by a test so that a fault would show)."""
    d = os.path.join(str(tmp_path), name)
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(d, "model.safetensors"), tensors, {"format": "pt"})
    return d

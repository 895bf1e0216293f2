"""Plain, slow, whole-sequence implementation of the Tudulix decoder.

The oracle of the Tudulix tests.  It shares no code with the ``prelude_b200``
package: it takes the parsed config.json and a ``dict`` of tensors keyed by
their safetensors names, runs a whole sequence at once with no cache, and
returns the logits of every position (and, on request, the residual stream
after every layer run).  One function per mechanism.

The design, in this file's notation (D = width, t = position from 0):

  norm        n(x; w) = x / sqrt(mean(x^2) + eps) * (1 + w)                (w stored around zero)
  start       e = scale * Embed[token] ;  r = e
  layer       r <- r + n1b(mixer(n1(r))) ;  r <- r + n2b(ff(n2(r)))        (the second half only where there is an ff)
  order       0 .. a-1, then (a .. b-1) n times, then b .. ; before every pass but the first r <- r + e
  mixers      'attention': grouped queries, window;  'latent_attention': one latent per token, window, gate
  ff          sum over the chosen experts x of p_x E_x(h), plus one expert that every token runs;
              E(h) = W_d [ a sigmoid(1.702 a) (b + 1) ],  a = min(W_g h, c),  b = clamp(W_u h, -c, c)
  output      logits = scale * W_head n_final(r)

All arithmetic is done in ``dtype`` (float64 by default); bfloat16 weights
convert exactly.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

ALPHA = 1.702


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_one(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * (1.0 + w)


# -- positions and masks ------------------------------------------------------------------------------------
def turn(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float, neighbours: bool) -> torch.Tensor:
    """x [T, heads, d]: pair i of the first ``dims`` entries turns by position * base^(-2i/dims); a pair is (2i, 2i + 1),
    or, without ``neighbours``, (i, i + dims/2)."""
    rate = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=x.dtype)
    ang = positions.to(x.dtype).reshape(-1, 1, 1) * rate
    a, b = (slice(0, dims, 2), slice(1, dims, 2)) if neighbours else (slice(0, dims // 2), slice(dims // 2, dims))
    out = x.clone()
    out[..., a] = x[..., a] * ang.cos() - x[..., b] * ang.sin()
    out[..., b] = x[..., b] * ang.cos() + x[..., a] * ang.sin()
    return out


def hidden_keys(T: int, window: Optional[int]) -> torch.Tensor:
    """[T, T] bool, row i: the keys that position i does not see."""
    back = torch.arange(T).reshape(-1, 1) - torch.arange(T).reshape(1, -1)
    hidden = back < 0
    return hidden if window is None else hidden | (back >= window)


def window_of(m: dict) -> Optional[int]:
    return None if m.get("mask") is None else m["mask"]["size"]


# -- grouped-query attention ----------------------------------------------------------------------------------
def grouped_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    at = torch.arange(T)
    q = turn((h @ w["q"].T).reshape(T, H, d), at, m["rot"]["dims"], m["rot"]["base"], True)
    k = turn((h @ w["k"].T).reshape(T, G, d), at, m["rot"]["dims"], m["rot"]["base"], True)
    v = (h @ w["v"].T).reshape(T, G, e)
    mine = torch.tensor([i // (H // G) for i in range(H)])
    s = torch.einsum("ihd,jhd->hij", q, k[:, mine]) * m["scale"]
    p = torch.softmax(s.masked_fill(hidden_keys(T, window_of(m)), -math.inf), dim=-1)
    return torch.einsum("hij,jhe->ihe", p, v[:, mine]).reshape(T, H * e) @ w["o"].T


# -- attention through one latent per token --------------------------------------------------------------------
def cached_rows(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
    """(latent [T, rank], turned key part [T, rot_dim]): what a token leaves for later ones."""
    T = h.shape[0]
    y = h @ w["dkv"].T
    c = rms(y[:, :m["kv_rank"]], eps) * w["dkv.norm"]
    kr = turn(y[:, m["kv_rank"]:].reshape(T, 1, -1), torch.arange(T), m["rot"]["dims"], m["rot"]["base"], False).reshape(T, -1)
    return c, kr


def latent_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, rows: Tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
    T = h.shape[0]
    H, d, e, rd = m["heads"], m["dim"], m["vdim"], m["rot_dim"]
    c, kr = rows
    q = (h @ w["q"].T).reshape(T, H, d + rd)
    q_rot = turn(q[..., d:], torch.arange(T), m["rot"]["dims"], m["rot"]["base"], False)
    k = (c @ w["uk"].T).reshape(T, H, d)
    v = (c @ w["uv"].T).reshape(T, H, e)
    s = (torch.einsum("ihd,jhd->hij", q[..., :d], k) + torch.einsum("ihd,jd->hij", q_rot, kr)) * m["scale"]
    p = torch.softmax(s.masked_fill(hidden_keys(T, window_of(m)), -math.inf), dim=-1)
    o = torch.einsum("hij,jhe->ihe", p, v).reshape(T, H * e)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# -- feed-forward ------------------------------------------------------------------------------------------------
def clamped_unit(a: torch.Tensor, b: torch.Tensor, limit: float) -> torch.Tensor:
    a, b = a.clamp(max=limit), b.clamp(-limit, limit)
    return a * torch.sigmoid(ALPHA * a) * (b + 1.0)


def expert(h: torch.Tensor, w: Dict[str, torch.Tensor], name: str, limit: float) -> torch.Tensor:
    return clamped_unit(h @ w[name + ".gate"].T, h @ w[name + ".up"].T, limit) @ w[name + ".down"].T


def route(logits: torch.Tensor, top: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """(experts [T, top], weights [T, top]): the largest logits, and the softmax over them alone."""
    best = logits.topk(top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def route_margin(logits: torch.Tensor, top: int) -> torch.Tensor:
    """[T]: the gap between the last chosen expert's logit and the best one's not chosen."""
    if top >= logits.shape[-1]:
        return torch.full((logits.shape[0],), math.inf, dtype=logits.dtype)
    ranked = logits.sort(dim=-1, descending=True).values
    return ranked[:, top - 1] - ranked[:, top]


def router_logits(h: torch.Tensor, w: Dict[str, torch.Tensor]) -> torch.Tensor:
    return h @ w["router"].T + w["router.b"]


def routed_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], mlp: dict) -> torch.Tensor:
    ids, p = route(router_logits(h, w), mlp["router"]["top"])
    out = torch.zeros_like(h)
    for x in range(mlp["router"]["experts"]):
        for c in range(ids.shape[1]):
            rows = (ids[:, c] == x).nonzero().reshape(-1)
            if rows.numel():
                out[rows] += p[rows, c].unsqueeze(-1) * expert(h[rows], w, f"e{x}", mlp["expert"]["limit"])
    if mlp.get("shared") is not None:
        out = out + expert(h, w, "shared", mlp["shared"]["limit"])
    return out


# -- the model -------------------------------------------------------------------------------------------------------
def sub(tensors: Dict[str, torch.Tensor], prefix: str, dtype) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(dtype) for k, v in tensors.items() if k.startswith(prefix)}


def run_order(cfg: dict) -> List[Tuple[int, bool]]:
    """(layer, whether the embedding output joins the stream right before it) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, False) for i in range(a)]
    for turn_no in range(loop["times"]):
        out += [(i, turn_no > 0 and i == a) for i in range(a, b)]
    return out + [(i, False) for i in range(b, n)]


def forward(cfg: dict, tensors: Dict[str, torch.Tensor], tokens, dtype=torch.float64, layers_out: Optional[list] = None,
            margins_out: Optional[List[torch.Tensor]] = None):
    """Logits [T, vocab] of a whole sequence; ``layers_out`` collects the residual stream after every layer run,
    ``margins_out`` every router's ``route_margin``."""
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return norm_around_one(x, tensors[name].to(dtype), eps)

    start = tensors["embed"].to(dtype)[torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    r = start
    for i, again in run_order(cfg):
        if again:
            r = r + start
        layer = cfg["layers"][i]
        m, w = layer["mixer"], sub(tensors, f"l{i}.mix.", dtype)
        h = norm(r, f"l{i}.norm1")
        if layer["type"] == "attention":
            y = grouped_attention(h, w, m)
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, w, m, cached_rows(h, w, m, eps))
        else:
            raise ValueError(f"unknown layer type {layer['type']!r}")
        r = r + norm(y, f"l{i}.norm1b")
        mlp = layer.get("mlp")
        if mlp is not None:
            w = sub(tensors, f"l{i}.mlp.", dtype)
            h = norm(r, f"l{i}.norm2")
            if margins_out is not None:
                margins_out.append(route_margin(router_logits(h, w), mlp["router"]["top"]))
            r = r + norm(routed_ff(h, w, mlp), f"l{i}.norm2b")
        if layers_out is not None:
            layers_out.append(r.clone())
    return norm(r, "final.norm") @ tensors["head"].to(dtype).T * cfg["logit_scale"]

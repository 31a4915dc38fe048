"""A plain, slow implementation of the Mumopel design, one function per mechanism, in torch on the CPU.

It shares no code with the package: it takes a configuration (the nested dict of ``config.json``) and a dict of
tensors by name and works on whole sequences.  Everything runs in the type of the tensors it is given (tests pass
float64).

Notation: W the width, T the tokens of one sequence, positions count from 0, X [S, T, W] the S streams,
ln(v) = (v - mean v) / sqrt(mean (v - mean v)^2 + eps) * w + b.
    sublayer   u = sum_s in_s X_s;  y = part(ln(u));  X_t <- sum_s mix_st X_s + out_t y
    layer      one sublayer with attention, one with the feed-forward (if there is one)
    output     l = E ln(sum_s X_s);  logits = cap tanh(l / cap)
"""
from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional

import torch


def layer_norm(v: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = v - v.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w + b


def rms_norm(v: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(dim=-1, keepdim=True) + eps) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------ streams --
def streams_read(X: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    """What a sublayer reads: sum over the streams of in_s X_s."""
    return torch.einsum("s,stw->tw", w_in, X)


def streams_write(X: torch.Tensor, mix: torch.Tensor, w_out: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """The streams behind a sublayer: stream t is sum_s mix[s, t] X_s + out_t y, all of them from the old ones."""
    return torch.einsum("sr,stw->rtw", mix, X) + w_out[:, None, None] * y[None]


# ------------------------------------------------------------------------------------------ attention --
def rotate_pairs(v: torch.Tensor, positions: torch.Tensor, rot: Optional[Mapping]) -> torch.Tensor:
    """v [T, heads, dim]; of the first rot.dims elements of every head, 2i turns with 2i + 1 by position * base^(-2i/dims)."""
    dims = int(rot["dims"]) if rot else 0
    if not dims:
        return v
    f = torch.tensor([float(rot["base"]) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(ang).to(v.dtype)[:, None, :], torch.sin(ang).to(v.dtype)[:, None, :]
    out = v.clone()
    a, b = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def chunk_mask(T: int, size: Optional[int]) -> torch.Tensor:
    """[T, T]: may position i (row) read position j?  j <= i, and both in the same chunk of ``size`` positions."""
    i = torch.arange(T)
    see = i[None, :] <= i[:, None]
    if size:
        see = see & (torch.div(i[None, :], size, rounding_mode="floor") == torch.div(i[:, None], size, rounding_mode="floor"))
    return see


def sink_softmax_attention(q, k, v, scale: float, see: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head h reads key/value head h // (H / G).  ``sink`` [H]: every
    softmax's denominator also holds exp(sink_h), as it is, without a key and without a value."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = torch.where(see, s, torch.full_like(s, -float("inf")))
        top = s.max(dim=1, keepdim=True).values
        if sink is not None:
            top = torch.maximum(top, sink[h].expand_as(top))
        e = torch.exp(s - top)
        den = e.sum(dim=1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - top)
        out[:, h] = (e / den) @ v[:, g]
    return out


def attention(h, w: Mapping[str, torch.Tensor], p: str, m: Mapping, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    pos = torch.arange(T)
    # one norm over all query heads together, one over all key heads together
    q = rms_norm(h @ w[p + ".q"].T, w[p + ".q.norm"], eps).view(T, H, d)
    k = rms_norm(h @ w[p + ".k"].T, w[p + ".k.norm"], eps).view(T, G, d)
    v = (h @ w[p + ".v"].T).view(T, G, dv)
    q, k = rotate_pairs(q, pos, m.get("rot")), rotate_pairs(k, pos, m.get("rot"))
    size = int(m["mask"]["size"]) if m.get("mask") else None
    o = sink_softmax_attention(q, k, v, float(m["scale"]), chunk_mask(T, size), w[p + ".sink"])
    return o.reshape(T, H * dv) @ w[p + ".o"].T


# ------------------------------------------------------------------------------------------ feed-forward --
def dense_ff(h, w, p: str) -> torch.Tensor:
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def clamped_expert(h, w, p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + ".gate"].T, max=limit)
    u = torch.clamp(h @ w[p + ".up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[p + ".down"].T


def route(h, w, p: str, r: Mapping):
    """(expert ids [T, top], weights [T, top]): the largest logits (bias included) and the softmax over those alone."""
    z = h @ w[p + ".router"].T + w[p + ".router.b"]
    top = z.topk(int(r["top"]), dim=-1)
    return top.indices, torch.softmax(top.values, dim=-1)


def moe_ff(h, w, p: str, ml: Mapping) -> torch.Tensor:
    ids, wts = route(h, w, p, ml["router"])
    out = torch.zeros_like(h)
    for e in range(int(ml["router"]["experts"])):
        t, c = (ids == e).nonzero(as_tuple=True)
        if t.numel():
            out[t] += wts[t, c][:, None] * clamped_expert(h[t], w, f"{p}.e{e}", float(ml["expert"]["limit"]))
    if ml.get("shared"):
        out = out + clamped_expert(h, w, p + ".shared", float(ml["shared"]["limit"]))
    return out


# ------------------------------------------------------------------------------------------ model --
def layer_order(cfg: Mapping) -> List[int]:
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    a, b = int(lp["start"]), int(lp["stop"])
    return list(range(a)) + list(range(a, b)) * int(lp["times"]) + list(range(b, n))


def forward(cfg: Mapping, w: Mapping[str, torch.Tensor], tokens: List[int], sums: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence; ``sums`` receives the sum of the streams after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    X = torch.stack([x] * int(cfg["streams"]))
    for i in layer_order(cfg):
        L, p = cfg["layers"][i], f"l{i}"
        ml = L.get("mlp")
        for q in (1, 2) if ml is not None else (1,):
            h = layer_norm(streams_read(X, w[f"{p}.hc{q}.in"]), w[f"{p}.norm{q}"], w[f"{p}.norm{q}.b"], eps)
            if q == 1:
                y = attention(h, w, p + ".mix", L["mixer"], eps)
            else:
                y = dense_ff(h, w, p + ".mlp") if ml["kind"] == "dense" else moe_ff(h, w, p + ".mlp", ml)
            X = streams_write(X, w[f"{p}.hc{q}.mix"], w[f"{p}.hc{q}.out"], y)
        if sums is not None:
            sums.append(X.sum(dim=0))
    z = layer_norm(X.sum(dim=0), w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T
    cap = float(cfg.get("logit_softcap") or 0.0)
    return cap * torch.tanh(z / cap) if cap else z


# ------------------------------------------------------------------------------------------ random weights --
def random_weights(cfg: Mapping, seed: int) -> Dict[str, torch.Tensor]:
    """Tensors of a model of ``cfg`` (float64, values that bfloat16 holds exactly), by name."""
    g = torch.Generator().manual_seed(seed)
    W, S = int(cfg["width"]), int(cfg["streams"])

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g, dtype=torch.float64) * std + mean).to(torch.bfloat16).double()

    def lin(out, inp, gain=1.0):
        return rnd(out, inp, std=gain / math.sqrt(inp))

    w = {"embed": rnd(int(cfg["vocab"]), W, std=0.6), "final.norm": rnd(W, std=0.2, mean=1.0), "final.norm.b": rnd(W, std=0.1)}
    for i, L in enumerate(cfg["layers"]):
        p, m, ml = f"l{i}", L["mixer"], L.get("mlp")
        H, G, d, dv = (int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        for q in (1, 2) if ml is not None else (1,):
            w[f"{p}.norm{q}"], w[f"{p}.norm{q}.b"] = rnd(W, std=0.2, mean=1.0), rnd(W, std=0.1)
            w[f"{p}.hc{q}.in"], w[f"{p}.hc{q}.out"] = rnd(S, std=0.3 / S, mean=1.0 / S), rnd(S, std=0.25, mean=0.5)
            # not symmetric, every stream fed by every other, and a size that neither dies nor grows over the layers
            w[f"{p}.hc{q}.mix"] = (0.8 * torch.eye(S, dtype=torch.float64) + rnd(S, S, std=0.1, mean=0.2 / S)).to(torch.bfloat16).double()
        a = p + ".mix"
        w[a + ".q"], w[a + ".k"], w[a + ".v"], w[a + ".o"] = lin(H * d, W), lin(G * d, W), lin(G * dv, W), lin(W, H * dv)
        w[a + ".q.norm"], w[a + ".k.norm"] = rnd(H * d, std=0.3, mean=1.0), rnd(G * d, std=0.3, mean=1.0)
        w[a + ".sink"] = rnd(H, std=1.5, mean=0.5)
        if ml is None:
            continue
        f = p + ".mlp"
        names = [(f, int(ml["ff"]))] if ml["kind"] == "dense" else \
            [(f"{f}.e{e}", int(ml["expert"]["ff"])) for e in range(int(ml["router"]["experts"]))] + \
            ([(f + ".shared", int(ml["shared"]["ff"]))] if ml.get("shared") else [])
        for n, F in names:
            w[n + ".gate"], w[n + ".up"], w[n + ".down"] = lin(F, W, 1.2), lin(F, W, 1.2), lin(W, F, 0.7)
        if ml["kind"] == "moe":
            E = int(ml["router"]["experts"])
            w[f + ".router"], w[f + ".router.b"] = lin(E, W), rnd(E, std=0.7)
    return w

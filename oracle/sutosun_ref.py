"""Slow reference of the Sutosun family in float64 on the CPU, one function per mechanism.

Test infrastructure only: nothing under agentic-traffic-testing_b200/ imports it, and it imports nothing from there.
Every function works on a whole sequence at once ([n, ...] tensors, position = row index) and is written as the
defining sums (a loop over positions for the recurrence, sums over all pairs of positions for attention; no pages, no
carried state, no chunks, no absorbed projections, no sorting of tokens by expert).

Notation: n tokens, model width W; `lin(u, M)` = u M^T for a matrix M [out, in]. `cfg` is the parsed config.json of a
model, `wt` maps tensor names to float64 tensors.

The family: x_t = rms(E[token_t]) w_embed; every layer is
    x <- x + mixer(rms(x) w1);      x <- x + ffn(rms(x) w2)        (ffn optional)
and may borrow all its tensors from another layer (`weights_of`). Three mixers: soft-max attention with grouped
key/value heads, biased projections, a norm over the whole q and the whole k projection and a query factor that grows
with the position (`attention`), linear attention with a fixed decay per head behind a rotation (`retention`), soft-max
attention whose keys and values are expanded from a cached latent, with a rotated part shared by all heads
(`latent_attention`). Both soft-max mixers have a learned sink per head. The feed-forward is dense with a tanh-gelu
gate or a mixture of silu-gated experts whose weights are the soft-max over the chosen, biased router outputs.
logits = cap tanh(W_head (rms(x) w_final) / cap).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional, Tuple

import torch

F64 = torch.float64


def lin(u: torch.Tensor, m: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = u @ m.T
    return y if b is None else y + b


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x divided by its root mean square over the last axis (eps under the root)."""
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return z / 2.0 * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def pair_frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> Tuple[torch.Tensor, float]:
    """f_i = base^(-2i/dims), i < dims/2, and the factor on cos and sin. With `scaling` (factor, original, fast, slow):
    a pair making t turns over `original` positions sits at index d(t) = dims ln(original / (2 pi t)) / (2 ln base);
    from lo = floor d(fast) (at least 0) to hi = ceil d(slow) (at most dims - 1) the frequency goes linearly from f_i to
    f_i / factor, and cos and sin are multiplied by 0.1 ln(factor) + 1."""
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    if not scaling:
        return f, 1.0
    factor, orig = float(scaling["factor"]), float(scaling["original"])

    def d(turns: float) -> float:
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(d(float(scaling["fast"]))), 0)
    hi = min(math.ceil(d(float(scaling["slow"]))), dims - 1)
    for i in range(dims // 2):
        s = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        f[i] = f[i] / factor * s + f[i] * (1.0 - s)
    return f, 0.1 * math.log(factor) + 1.0


def rotate_halves(x: torch.Tensor, freqs: torch.Tensor, mag: float = 1.0) -> torch.Tensor:
    """x [n, ..., D]: of its first 2m elements (m = len(freqs)) element i and element i + m at position p are turned by
    p f_i (and scaled by mag); the others stay."""
    n, m = x.shape[0], freqs.shape[0]
    ang = torch.arange(n, dtype=F64)[:, None] * freqs[None, :]
    shape = [n] + [1] * (x.dim() - 2) + [m]
    co, si = (torch.cos(ang) * mag).view(shape), (torch.sin(ang) * mag).view(shape)
    out = x.clone()
    u, v = x[..., :m], x[..., m:2 * m]
    out[..., :m] = u * co - v * si
    out[..., m:2 * m] = v * co + u * si
    return out


def query_factor(n: int, coef: float, every: float) -> torch.Tensor:
    """1 + coef ln(floor((p + 1) / every) + 1) for p = 0 .. n - 1."""
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in range(n)], dtype=F64)


def sink_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, sink: torch.Tensor) -> torch.Tensor:
    """q [n, H, D], k [n, G, D], v [n, G, V]; head h reads key/value head h // (H / G). The weights of the keys j <= i are
    exp(score) over their sum plus exp(sink_h)."""
    n, H, _ = q.shape
    G = k.shape[1]
    kk = k.repeat_interleave(H // G, dim=1)
    vv = v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale
    s = s.masked_fill(torch.ones(n, n, dtype=torch.bool).triu(1)[None], float("-inf"))
    m = torch.maximum(s.max(-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - m)
    w = e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - m))
    return torch.einsum("hij,jhv->ihv", w, vv)


def attention_mixer(u: torch.Tensor, c: dict, wt: Dict[str, torch.Tensor], m: str, eps: float) -> torch.Tensor:
    H, G, D, V = int(c["heads"]), int(c["kv_heads"]), int(c["dim"]), int(c["vdim"])
    n = u.shape[0]
    q = unit_rms(lin(u, wt[m + "q"], wt[m + "q.b"]), eps) * wt[m + "q.norm"]
    k = unit_rms(lin(u, wt[m + "k"], wt[m + "k.b"]), eps) * wt[m + "k.norm"]
    v = lin(u, wt[m + "v"], wt[m + "v.b"])
    qt = c.get("q_temp")
    if qt:
        q = q * query_factor(n, float(qt["coef"]), float(qt["every"]))[:, None]
    o = sink_attention(q.view(n, H, D), k.view(n, G, D), v.view(n, G, V), float(c["scale"]), wt[m + "sink"])
    o = o * torch.sigmoid(lin(u, wt[m + "g"]))[:, :, None]
    return lin(o.reshape(n, H * V), wt[m + "o"])


def decayed_outer_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: float) -> torch.Tensor:
    """One head. S_t = decay S_(t-1) + k_t v_t^T from S = 0, o_t = S_t^T q_t."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out, 0)


def decayed_pair_sum(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: float) -> torch.Tensor:
    """The same as a sum over pairs: o_t = sum_(s <= t) decay^(t - s) (q_t . k_s) v_s."""
    n = q.shape[0]
    d = torch.arange(n, dtype=F64)
    w = torch.pow(torch.tensor(float(decay), dtype=F64), (d[:, None] - d[None, :]).clamp(min=0.0)).tril()
    return (w * (q @ k.T)) @ v


def retention_mixer(u: torch.Tensor, c: dict, wt: Dict[str, torch.Tensor], m: str, eps: float) -> torch.Tensor:
    H, D, V = int(c["heads"]), int(c["dim"]), int(c["vdim"])
    n = u.shape[0]
    q, k = lin(u, wt[m + "q"]).view(n, H, D), lin(u, wt[m + "k"]).view(n, H, D)
    v = lin(u, wt[m + "v"]).view(n, H, V)
    rot = c.get("rot") or {}
    if rot.get("dims"):
        f, mag = pair_frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
        q, k = rotate_halves(q, f, mag), rotate_halves(k, f, mag)
    k = k * D ** -0.5
    o = torch.stack([decayed_outer_recurrence(q[:, h], k[:, h], v[:, h], float(c["decay"][h])) for h in range(H)], 1)
    return lin(unit_rms(o, eps).reshape(n, H * V) * silu(lin(u, wt[m + "g"])), wt[m + "o"])


def latent_mixer(u: torch.Tensor, c: dict, wt: Dict[str, torch.Tensor], m: str, eps: float) -> torch.Tensor:
    """Queries per head [D plain | R rotated]; keys [W_uk c | one rotated part for all heads], values W_uv c."""
    H, D, R, V, C = (int(c[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    n = u.shape[0]
    q = lin(u, wt[m + "q"]).view(n, H, D + R)
    z = lin(u, wt[m + "dkv"])
    lat, kr = unit_rms(z[:, :C], eps) * wt[m + "dkv.norm"], z[:, C:]
    rot = c.get("rot") or {}
    if R and rot.get("dims"):
        f, mag = pair_frequencies(int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
        q = torch.cat([q[..., :D], rotate_halves(q[..., D:], f, mag)], -1)
        kr = rotate_halves(kr, f, mag)
    k = torch.cat([lin(lat, wt[m + "uk"]).view(n, H, D), kr[:, None, :].expand(n, H, R)], -1)
    v = lin(lat, wt[m + "uv"]).view(n, H, V)
    o = sink_attention(q, k, v, float(c["scale"]), wt[m + "sink"])
    return lin(o.reshape(n, H * V), wt[m + "o"])


def dense_gelu(u: torch.Tensor, wt: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(gelu_tanh(lin(u, wt[p + "gate"])) * lin(u, wt[p + "up"]), wt[p + "down"])


def silu_expert(u: torch.Tensor, wt: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(silu(lin(u, wt[p + "gate"])) * lin(u, wt[p + "up"]), wt[p + "down"])


def route(u: torch.Tensor, router: torch.Tensor, bias: torch.Tensor, top: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """Chosen experts [n, top] (the largest biased outputs) and their weights: the soft-max over the chosen outputs."""
    val, idx = torch.topk(lin(u, router, bias), top, dim=-1)
    return idx, torch.softmax(val, -1)


def expert_mixture(u: torch.Tensor, c: dict, wt: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    idx, wgt = route(u, wt[p + "router"], wt[p + "router.b"], int(c["router"]["top"]))
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(idx.shape[1]):
            y[t] += wgt[t, j] * silu_expert(u[t:t + 1], wt, f"{p}e{int(idx[t, j])}.")[0]
    return y


MIXERS = {"attention": attention_mixer, "retention": retention_mixer, "latent_attention": latent_mixer}


def forward(cfg: dict, wt: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab] of one sequence; `residuals`, if a list, receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = unit_rms(wt["embed"][tokens], eps) * wt["embed.norm"]
    for i, l in enumerate(cfg["layers"]):
        p = f"l{int(l.get('weights_of', i))}."
        x = x + MIXERS[l["type"]](unit_rms(x, eps) * wt[p + "norm1"], l["mixer"], wt, p + "mix.", eps)
        mlp = l.get("mlp")
        if mlp is not None:
            u = unit_rms(x, eps) * wt[p + "norm2"]
            x = x + (dense_gelu(u, wt, p + "mlp.") if mlp["kind"] == "dense" else expert_mixture(u, mlp, wt, p + "mlp."))
        if residuals is not None:
            residuals.append(x.clone())
    z = lin(unit_rms(x, eps) * wt["final.norm"], wt["head"])
    cap = float(cfg["logit_softcap"])
    return cap * torch.tanh(z / cap)


# ---- checkpoints for tests --------------------------------------------------------------------------------------------


def checkpoint_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    W, out = int(cfg["width"]), {}
    out["embed"], out["embed.norm"] = (int(cfg["vocab"]), W), (W,)
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        p, c, m = f"l{i}.", l["mixer"], f"l{i}.mix."
        H, D, V = int(c["heads"]), int(c["dim"]), int(c["vdim"])
        out[p + "norm1"] = (W,)
        if l["type"] == "attention":
            G = int(c["kv_heads"])
            for nm, r in (("q", H * D), ("k", G * D), ("v", G * V)):
                out[m + nm], out[m + nm + ".b"] = (r, W), (r,)
            out.update({m + "q.norm": (H * D,), m + "k.norm": (G * D,), m + "sink": (H,), m + "g": (H, W), m + "o": (W, H * V)})
        elif l["type"] == "retention":
            out.update({m + "q": (H * D, W), m + "k": (H * D, W), m + "v": (H * V, W), m + "g": (H * V, W), m + "o": (W, H * V)})
        else:
            R, C = int(c["rot_dim"]), int(c["kv_rank"])
            out.update({m + "q": (H * (D + R), W), m + "dkv": (C + R, W), m + "dkv.norm": (C,), m + "uk": (H * D, C),
                        m + "uv": (H * V, C), m + "sink": (H,), m + "o": (W, H * V)})
        mlp = l.get("mlp")
        if mlp is None:
            continue
        out[p + "norm2"] = (W,)
        f = p + "mlp."
        if mlp["kind"] == "dense":
            F = int(mlp["ff"])
            out.update({f + "gate": (F, W), f + "up": (F, W), f + "down": (W, F)})
        else:
            E, F = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
            for e in range(E):
                out.update({f"{f}e{e}.gate": (F, W), f"{f}e{e}.up": (F, W), f"{f}e{e}.down": (W, F)})
            out[f + "router"], out[f + "router.b"] = (E, W), (E,)
    out["final.norm"], out["head"] = (W,), (int(cfg["vocab"]), W)
    return out


def random_checkpoint(cfg: dict, seed: int, round_bf16: bool = True) -> Dict[str, torch.Tensor]:
    """Seeded float64 tensors (rounded to bf16 values, so that a bf16 copy of them is exact)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, sh in checkpoint_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        t = torch.randn(sh, generator=g, dtype=F64)
        if name.endswith("router.b"):
            t = 0.5 * t
        elif leaf == "b":
            t = 0.3 * t
        elif leaf == "sink":
            t = 1.0 + t
        elif name == "embed":
            t = 0.7 * t
        elif len(sh) == 2:
            t = t * (sh[1] ** -0.5) * (2.0 if leaf in ("router", "head") else 1.0)
        else:
            t = 1.0 + 0.1 * t
        out[name] = t.to(torch.bfloat16).to(F64) if round_bf16 else t
    return out

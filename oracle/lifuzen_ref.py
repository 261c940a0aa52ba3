"""Slow reference of the Lifuzen family in float64 on the CPU, one function per mechanism.

Test infrastructure only: nothing under agentic-traffic-testing_b200/ imports it, and it imports nothing from there.
Every function works on a whole sequence at once ([n, ...] tensors, position = row index) and is written as the
defining sums (a loop over positions for the recurrence, sums over all pairs of positions for attention; no pages, no
carried state, no chunks, no sorting of tokens by expert).

Notation: n tokens, model width W; `lin(u, M)` = u M^T for a matrix M [out, in]. `cfg` is the parsed config.json of a
model, `wt` maps tensor names to float64 tensors.

The family: x_t = E[token_t]; every layer is parallel, x <- x + m (mixer(nrm(x, w1)) + ffn(nrm(x, w2))), ffn optional, with
nrm(x, w) = x / rms(x) * (1 + w). A block of layers may run several times; before a pass x gains the embedding output (all
passes but the first) and a vector of its own. Mixers: a selective state-space recurrence with its gate in front of a grouped
norm, and soft-max attention whose queries and keys pass a short causal convolution, whose values are the convolved keys
themselves, with a sink of score 0. Feed-forward: a mixture of squared-ReLU experts with sigmoid scores, each chosen expert
reading its input times its score. logits = cap tanh(E nrm(x, w) / cap).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

F64 = torch.float64


def lin(u: torch.Tensor, m: torch.Tensor) -> torch.Tensor:
    return u @ m.T


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def swish(x: torch.Tensor) -> torch.Tensor:
    return x / (1.0 + torch.exp(-x))


def causal_taps(u: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """y_t[c] = bias[c] + sum_j w[c, j] u_(t - K + 1 + j)[c] with K = w.shape[1]; rows before the sequence are zero."""
    n, K = u.shape[0], w.shape[1]
    y = torch.zeros_like(u) if bias is None else bias.expand(n, -1).clone()
    for t in range(n):
        for j in range(K):
            s = t - K + 1 + j
            if s >= 0:
                y[t] = y[t] + w[:, j] * u[s]
    return y


def rotate_pairs(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [n, heads, D]: the pair (2i, 2i + 1), i < dims/2, of the row at position p turns by p base^(-2i/dims)."""
    out = x.clone()
    p = torch.arange(x.shape[0], dtype=F64)[:, None]
    for i in range(dims // 2):
        a = p * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def sink_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q [n, H, D], k [n, G, D], v [n, G, V]; query head h reads key/value head h // (H / G). Causal; weights
    exp(s_j) / (1 + sum exp(s_j)): the extra 1 is a sink of score 0 that carries no value."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(torch.arange(n)[None, :] > torch.arange(n)[:, None], float("-inf"))
        top = s.max(-1, keepdim=True).values.clamp(min=0.0)          # common factor exp(-top) in numerator and denominator
        e = torch.exp(s - top)
        out[:, h] = (e / (torch.exp(-top) + e.sum(-1, keepdim=True))) @ v[:, g]
    return out


def attention_mixer(u: torch.Tensor, c: dict, wt: Dict[str, torch.Tensor], m: str, eps: float) -> torch.Tensor:
    n = u.shape[0]
    H, G, D = int(c["heads"]), int(c["kv_heads"]), int(c["dim"])
    q = causal_taps(lin(u, wt[m + "q"]), wt[m + "q.conv"]).view(n, H, D)
    k = causal_taps(lin(u, wt[m + "k"]), wt[m + "k.conv"]).view(n, G, D)
    v = k
    rot = c.get("rot") or {}
    rd = int(rot.get("dims", 0) or 0)
    if rd:
        q, k = (rotate_pairs(x, rd, float(rot["base"])) for x in (q, k))
    o = sink_attention(unit_rms(q, eps), unit_rms(k, eps), v, float(c["scale"]))
    return lin(o.reshape(n, H * D), wt[m + "o"])


def selective_scan(x: torch.Tensor, b: torch.Tensor, c: torch.Tensor, dt: torch.Tensor, a_log: torch.Tensor,
                   skip: torch.Tensor) -> torch.Tensor:
    """x [n, H, P], b / c [n, G, N], dt [n, H]: per head S_t = exp(-exp(A_log) dt) S_(t-1) + dt b_t x_t^T,
    y_t = S_t^T c_t + skip x_t, head h reading group h // (H / G)."""
    n, H, P = x.shape
    G, N = b.shape[1], b.shape[2]
    y = torch.zeros(n, H, P, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        S = torch.zeros(N, P, dtype=F64)
        for t in range(n):
            S = torch.exp(-torch.exp(a_log[h]) * dt[t, h]) * S + dt[t, h] * b[t, g][:, None] * x[t, h][None, :]
            y[t, h] = S.T @ c[t, g] + skip[h] * x[t, h]
    return y


def softplus(x: torch.Tensor) -> torch.Tensor:
    return x.clamp(min=0.0) + torch.log1p(torch.exp(-x.abs()))


def mamba2_mixer(u: torch.Tensor, c: dict, wt: Dict[str, torch.Tensor], m: str, eps: float) -> torch.Tensor:
    n = u.shape[0]
    H, P, N, G, R = (int(c[k]) for k in ("heads", "vdim", "state", "groups", "norm_groups"))
    inner = H * P
    z, xbc, dt = torch.split(lin(u, wt[m + "in"]), [inner, inner + 2 * G * N, H], dim=-1)
    x, b, cc = torch.split(swish(causal_taps(xbc, wt[m + "conv"], wt[m + "conv.b"])), [inner, G * N, G * N], dim=-1)
    y = selective_scan(x.view(n, H, P), b.view(n, G, N), cc.view(n, G, N), softplus(dt + wt[m + "dt_bias"]), wt[m + "A_log"],
                       wt[m + "D"]).reshape(n, inner)
    y = unit_rms((y * swish(z)).view(n, R, inner // R), eps).reshape(n, inner) * wt[m + "norm"]
    return lin(y, wt[m + "o"])


def squared_relu_expert(u: torch.Tensor, wt: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(lin(u, wt[p + "up"]).clamp(min=0.0) ** 2, wt[p + "down"])


def route(u: torch.Tensor, router: torch.Tensor, top: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """Chosen experts [n, top] and their scores: sigmoids, the `top` largest, as they are."""
    s = 1.0 / (1.0 + torch.exp(-lin(u, router)))
    val, idx = torch.topk(s, top, dim=-1)
    return idx, val


def expert_mixture(u: torch.Tensor, f: dict, wt: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    idx, wgt = route(u, wt[p + "router"], int(f["router"]["top"]))
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(idx.shape[1]):
            y[t] = y[t] + squared_relu_expert(wgt[t, j] * u[t:t + 1], wt, f"{p}e{int(idx[t, j])}.")[0]
    return y


def soft_cap(z: torch.Tensor, cap: Optional[float]) -> torch.Tensor:
    return cap * torch.tanh(z / cap) if cap else z


def execution_order(cfg: dict) -> List[Tuple[int, Optional[int]]]:
    """(layer, pass number or None) in the order of execution."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    out: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(a)]
    for t in range(times):
        out += [(i, t) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def forward(cfg: dict, wt: Dict[str, torch.Tensor], tokens: List[int], residuals: Optional[list] = None) -> torch.Tensor:
    """Logits [n, vocab] of one sequence; `residuals`, if a list, receives the stream after every layer run."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg.get("residual_mult", 1.0))
    x0 = wt["embed"][tokens]
    x = x0.clone()
    for i, t in execution_order(cfg):
        if t is not None and i == int(cfg["loop"]["start"]):
            x = (x + x0 if t > 0 else x) + wt["loop.step"][t]
        l, p = cfg["layers"][i], f"l{i}."
        mix = {"attention": attention_mixer, "mamba2": mamba2_mixer}[l["type"]]
        y = mix(centred_norm(x, wt[p + "norm1"], eps), l["mixer"], wt, p + "mix.", eps)
        if l.get("mlp") is not None:
            y = y + expert_mixture(centred_norm(x, wt[p + "norm2"], eps), l["mlp"], wt, p + "mlp.")
        x = x + mult * y
        if residuals is not None:
            residuals.append(x.clone())
    return soft_cap(lin(centred_norm(x, wt["final.norm"], eps), wt["embed"]), cfg.get("logit_softcap"))


# ---- checkpoints for tests --------------------------------------------------------------------------------------------


def checkpoint_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    W, out = int(cfg["width"]), {}
    out["embed"] = (int(cfg["vocab"]), W)
    if cfg.get("loop"):
        out["loop.step"] = (int(cfg["loop"]["times"]), W)
    for i, l in enumerate(cfg["layers"]):
        p, c, m = f"l{i}.", l["mixer"], f"l{i}.mix."
        out[p + "norm1"] = (W,)
        H, K = int(c["heads"]), int(c["conv"])
        if l["type"] == "attention":
            G, D = int(c["kv_heads"]), int(c["dim"])
            out.update({m + "q": (H * D, W), m + "k": (G * D, W), m + "q.conv": (H * D, K), m + "k.conv": (G * D, K),
                        m + "o": (W, H * D)})
        else:
            P, N, G = int(c["vdim"]), int(c["state"]), int(c["groups"])
            inner, ch = H * P, H * P + 2 * G * N
            out.update({m + "in": (inner + ch + H, W), m + "conv": (ch, K), m + "conv.b": (ch,), m + "dt_bias": (H,),
                        m + "A_log": (H,), m + "D": (H,), m + "norm": (inner,), m + "o": (W, inner)})
        f = l.get("mlp")
        if f is not None:
            F, E = int(f["expert"]["ff"]), int(f["router"]["experts"])
            out[p + "norm2"] = (W,)
            for e in range(E):
                out[f"{p}mlp.e{e}.up"], out[f"{p}mlp.e{e}.down"] = (F, W), (W, F)
            out[p + "mlp.router"] = (E, W)
    out["final.norm"] = (W,)
    return out


def random_checkpoint(cfg: dict, seed: int, round_bf16: bool = True) -> Dict[str, torch.Tensor]:
    """Seeded float64 tensors (rounded to bf16 values, so that a bf16 copy of them is exact)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, sh in checkpoint_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        r = torch.randn(sh, generator=g, dtype=F64)
        if leaf == "conv":
            t = 0.35 * r
        elif leaf == "A_log":
            t = torch.log(0.3 + 3.0 * torch.rand(sh, generator=g, dtype=F64))
        elif leaf == "dt_bias":
            t = -2.0 + r
        elif leaf == "D" or name.endswith("mix.norm"):
            t = 1.0 + 0.2 * r
        elif name == "embed":
            t = r
        elif name == "loop.step":
            t = 0.5 * r
        elif len(sh) == 2:
            gain = 2.5 if leaf == "router" else (1.6 if leaf in ("up", "down") else 1.0)
            t = r * (sh[1] ** -0.5) * gain
        else:
            t = 0.2 * r          # norm weights (stored around zero), the convolution's bias
        out[name] = t.to(torch.bfloat16).to(F64) if round_bf16 else t
    return out

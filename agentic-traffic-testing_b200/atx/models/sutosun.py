"""Sutosun: a decoder-only family whose layers are listed one by one in config.json, each with a norm in front of its sublayers:

    x_t = rms(embed[token_t]) w_embed                       rms(x) = x / sqrt(mean(x^2) + eps)
    x  <- x + mixer(rms(x) w1)
    x  <- x + ffn(rms(x) w2)                                                                   (ffn optional)
    logits = cap tanh(head . (rms(x) w_final) / cap)

A layer with `weights_of: j` has no tensors of its own: it runs layer j's with pages or a state of its own. Three mixers:

* `attention`: soft-max attention with grouped key/value heads; q, k and v have biases; RMS norm over the whole q and the whole k
  projection; no rotation, positions enter through a query factor 1 + coef ln(floor((p + 1) / every) + 1); a learned sink per head
  in the denominator; sigmoid(W_g u) per head on the output.
* `retention`: linear attention with a fixed decay per head, S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, behind a rotation
  (pairs half the rotated range apart) of q and k and dim^(-1/2) on k; every head's output is divided by its root mean square,
  multiplied by silu(W_g u) and projected.
* `latent_attention`: soft-max attention over a cached latent, per head [dim plain | rot_dim rotated] queries straight from W_q;
  W_dkv gives [latent (normed) | one rotated key part shared by all heads]; keys W_uk c, values W_uv c; frequencies stretched by
  pair index and a magnitude on cos / sin; a learned sink per head. Runs in the absorbed form: only the latent row is cached, the
  query of head h becomes [W_uk,h^T q_plain | rotated q part], attention runs as ONE key/value head shared by all query heads whose
  value is the row's leading kv_rank elements, and W_uv,h is applied to the head's result.

The feed-forward is dense, W_down (gelu(W_gate x) * W_up x) with the tanh form of gelu, or a mixture of experts with silu gates: the
`top` largest biased router outputs are chosen and weighted by the soft-max over the chosen ones alone.

State besides the pages, per live sequence (a state slot): the [heads, dim, vdim] fp32 state of every retention layer.

fp32 whatever the element type: the residual stream (the GEMMs of the output and down projections add into it), every norm, rotation,
the query factor, scores and weights of the attention, the recurrence and its state, router outputs and weights, the weighted sum,
the logit cap. Projections run in the element type (bf16 on the tcgen05 GEMM and the tensor-core head / expert products, or fp32 on
the FMA pipe) with fp32 accumulation.

The program below only issues kernels; scheduling, pages, state slots, staging, sampling and the step loop are the runner's
and the engine's (atx/runner.py, atx/engine.py)."""
from __future__ import annotations

import ctypes
import json
import math
from dataclasses import dataclass, field
from pathlib import Path
from typing import Dict, List, Optional, Tuple

import torch

from .. import _cabi
from .common import Experts, PagedAttention, _Linear, gate_up_matrix, rotation_table_scaled, stretched_frequencies

MIXERS = ("attention", "retention", "latent_attention")

# ---- configuration --------------------------------------------------------------------------------------------------


def _rot_key(c: dict) -> Optional[tuple]:
    rot = c.get("rot") or {}
    dims = int(rot.get("dims", 0) or 0)
    if not dims:
        return None
    sc = rot.get("scaling") or None
    return (float(rot["base"]), dims, tuple(float(sc[k]) for k in ("factor", "original", "fast", "slow")) if sc else None)


@dataclass
class Config:
    name: str = "sutosun"
    vocab_size: int = 0
    width: int = 0
    eps: float = 1e-6
    logit_softcap: float = 0.0                         # 0: logits as they are
    layers: List[dict] = field(default_factory=list)   # {"type", "mixer", "mlp", "weights_of"} as in config.json
    eos_token_ids: tuple = ()
    bos_token_id: int = 0
    max_position_embeddings: int = 131072    # the design sets no limit; this bounds the server's default max_model_len
    architecture = "Sutosun"

    @classmethod
    def from_json(cls, d: dict, name: str = "sutosun") -> "Config":
        cfg = cls(name=name, vocab_size=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]),
                  logit_softcap=float(d.get("logit_softcap") or 0.0), layers=[json.loads(json.dumps(l)) for l in d["layers"]])
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.logit_softcap < 0:
            raise ValueError(f"logit_softcap={self.logit_softcap} must not be negative")
        for i, l in enumerate(self.layers):
            if l["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            c = l["mixer"] = dict(l["mixer"])
            c.setdefault("vdim", c["dim"])
            rk = _rot_key(c)
            if l["type"] == "attention":
                c.setdefault("kv_heads", c["heads"])
                if c["heads"] % c["kv_heads"]:
                    raise ValueError(f"layer {i}: {c['heads']} heads over {c['kv_heads']} key/value heads")
                if c.get("q_temp") and float(c["q_temp"]["every"]) <= 0:
                    raise ValueError(f"layer {i}: q_temp.every must be positive")
            elif l["type"] == "retention":
                if len(c["decay"]) != c["heads"]:
                    raise ValueError(f"layer {i}: {len(c['decay'])} decays for {c['heads']} heads")
                if rk is not None and (rk[1] % 2 or rk[1] > c["dim"]):
                    raise ValueError(f"layer {i}: rot.dims={rk[1]} must be even and at most dim={c['dim']}")
            else:
                c.setdefault("rot_dim", 0)
                if c["rot_dim"] and (rk is None or rk[1] % 2 or rk[1] > c["rot_dim"]):
                    raise ValueError(f"layer {i}: rot.dims must be even and at most rot_dim={c['rot_dim']}")
            mlp = l.get("mlp")
            if mlp is not None:
                kind = mlp.get("kind", "dense")
                if kind == "moe":
                    r = mlp["router"]
                    if not 0 < int(r["top"]) <= int(r["experts"]):
                        raise ValueError(f"layer {i}: top={r['top']} of {r['experts']} experts")
                elif kind != "dense":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")
        for i, l in enumerate(self.layers):
            if l.get("weights_of") is None:
                continue
            j, seen = i, {i}
            while self.layers[j].get("weights_of") is not None:
                j = int(self.layers[j]["weights_of"])
                if not 0 <= j < len(self.layers) or j in seen:
                    raise ValueError(f"layer {i}: weights_of={l['weights_of']} must lead to a layer with tensors of its own")
                seen.add(j)
            o = self.layers[j]
            if (o["type"], o["mixer"], o.get("mlp")) != (l["type"], l["mixer"], l.get("mlp")):
                raise ValueError(f"layer {i}: uses layer {j}'s tensors but differs from it")

    def source(self, i: int) -> int:
        """The layer whose tensors layer i runs."""
        while self.layers[i].get("weights_of") is not None:
            i = int(self.layers[i]["weights_of"])
        return i

    @property
    def recurrent(self) -> bool:
        """A state slot per sequence: the states of the retention layers."""
        return any(l["type"] == "retention" for l in self.layers)

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def layer_shapes(self, i: int) -> Dict[str, Tuple[int, ...]]:
        W, l, p, m, out = self.width, self.layers[i], f"l{i}.", f"l{i}.mix.", {}
        c = l["mixer"]
        H, D, V = int(c["heads"]), int(c["dim"]), int(c["vdim"])
        out[p + "norm1"] = (W,)
        if l["type"] == "attention":
            G = int(c["kv_heads"])
            out.update({m + "q": (H * D, W), m + "q.b": (H * D,), m + "k": (G * D, W), m + "k.b": (G * D,), m + "v": (G * V, W),
                        m + "v.b": (G * V,), m + "q.norm": (H * D,), m + "k.norm": (G * D,), m + "sink": (H,), m + "g": (H, W),
                        m + "o": (W, H * V)})
        elif l["type"] == "retention":
            out.update({m + "q": (H * D, W), m + "k": (H * D, W), m + "v": (H * V, W), m + "g": (H * V, W), m + "o": (W, H * V)})
        else:
            R, C = int(c["rot_dim"]), int(c["kv_rank"])
            out.update({m + "q": (H * (D + R), W), m + "dkv": (C + R, W), m + "dkv.norm": (C,), m + "uk": (H * D, C),
                        m + "uv": (H * V, C), m + "sink": (H,), m + "o": (W, H * V)})
        mlp = l.get("mlp")
        if mlp is not None:
            f = p + "mlp."
            out[p + "norm2"] = (W,)
            if mlp.get("kind", "dense") == "dense":
                F = int(mlp["ff"])
                out.update({f + "gate": (F, W), f + "up": (F, W), f + "down": (W, F)})
            else:
                E, F = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
                for e in range(E):
                    out.update({f"{f}e{e}.gate": (F, W), f"{f}e{e}.up": (F, W), f"{f}e{e}.down": (W, F)})
                out.update({f + "router": (E, W), f + "router.b": (E,)})
        return out

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every tensor of a checkpoint of this configuration."""
        out = {"embed": (self.vocab_size, self.width), "embed.norm": (self.width,)}
        for i in range(len(self.layers)):
            if self.source(i) == i:
                out.update(self.layer_shapes(i))
        out["final.norm"], out["head"] = (self.width,), (self.vocab_size, self.width)
        return out

    # ---- bytes, for the benchmarks' rooflines -------------------------------------------------------------------
    def weight_bytes_per_decode_step(self, elem: int = 2, tokens: int = 1) -> int:
        """Weight bytes a decode step of `tokens` tokens streams: every layer's matrices each time it runs, the output head; of the
        experts at most tokens * top per layer."""
        n = self.vocab_size * self.width
        for i, l in enumerate(self.layers):
            n += sum(math.prod(v) for k, v in self.layer_shapes(self.source(i)).items() if ".mlp.e" not in k)
            mlp = l.get("mlp")
            if mlp is not None and mlp.get("kind") == "moe":
                r = mlp["router"]
                n += min(int(r["experts"]), tokens * int(r["top"])) * 3 * int(mlp["expert"]["ff"]) * self.width
        return elem * n

    def kv_bytes_per_token(self, elem: int = 2) -> int:
        n = 0
        for l in self.layers:
            c = l["mixer"]
            if l["type"] == "attention":
                n += int(c["kv_heads"]) * (int(c["dim"]) + int(c["vdim"]))
            elif l["type"] == "latent_attention":
                n += int(c["kv_rank"]) + int(c["rot_dim"])
        return n * elem

    def state_bytes_per_sequence(self) -> int:
        return 4 * sum(int(l["mixer"]["heads"]) * int(l["mixer"]["dim"]) * int(l["mixer"]["vdim"]) for l in self.layers
                       if l["type"] == "retention")

    def decode_kv_bytes(self, ctx: int, elem: int = 2) -> int:
        """Page bytes one decoded token at context length ctx reads."""
        return ctx * self.kv_bytes_per_token(elem)


def named_shape(name: str) -> Optional[Config]:
    """`random:sutosun-<size>`: shapes whose layers resemble a real model's, for benchmarks (no checkpoint exists).
    `sutosun-8b` / `sutosun-1b` have the width, feed-forward size, vocabulary and depth of the Llama 8B / 1B shapes; layers in the
    pattern retention + dense feed-forward, latent attention + experts, attention + experts, retention + dense feed-forward."""
    key = name.lower()
    shapes = {"sutosun-8b": (4096, 14336, 8, 128256), "sutosun-1b": (2048, 8192, 4, 128256),
              "sutosun-tiny": (256, 512, 1, 1024)}     # width, feed-forward, repeats of the 4-layer pattern, vocabulary
    if key not in shapes:
        return None
    W, F, groups, vocab = shapes[key]
    hd = 128 if W >= 4096 else 64
    heads = W // hd
    moe = {"kind": "moe", "expert": {"ff": max(64, F // 4 // 64 * 64)}, "router": {"experts": 8, "top": 2}}
    dense = {"kind": "dense", "ff": F}
    ret = {"decay": [1.0 - 2.0 ** -(5.0 + 5.0 * h / max(1, heads - 1)) for h in range(heads)], "dim": hd, "heads": heads, "vdim": hd,
           "rot": {"base": 10000.0, "dims": hd}}
    lat = {"dim": hd, "heads": heads, "vdim": hd, "kv_rank": 128, "rot_dim": 64, "scale": (hd + 64) ** -0.5,
           "rot": {"base": 500000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}}}
    att = {"dim": hd, "heads": heads, "kv_heads": max(1, heads // 4), "vdim": hd, "scale": hd ** -0.5,
           "q_temp": {"coef": 0.1, "every": 8192}}
    layers = [{"type": "retention", "mixer": ret, "mlp": dense}, {"type": "latent_attention", "mixer": lat, "mlp": moe},
              {"type": "attention", "mixer": att, "mlp": moe}, {"type": "retention", "mixer": ret, "mlp": dense}]
    cfg = Config(name=key, vocab_size=vocab, width=W, eps=1e-6, logit_softcap=30.0, layers=json.loads(json.dumps(layers * groups)))
    cfg.validate()
    return cfg


# ---- weights ----------------------------------------------------------------------------------------------------------


class _Layer:
    """Device tensors of one layer in the layout the kernels read (projections that share an input are stacked)."""

    def __init__(self) -> None:
        self.kind = ""
        self.norm1 = self.norm2 = None
        self.w_in = self.w_o = None          # attention: [q | k | v | g]; retention: [q | k | v | g]; latent: [q | dkv]
        self.bq = self.bk = self.bv = self.q_norm = self.k_norm = None   # attention
        self.sinks = None                    # fp32 [heads]
        self.decay = None                    # retention: fp32 [heads]
        self.dkv_norm = self.w_ukt = self.w_uv = None   # latent: [heads * kv_rank, dim] (W_uk per head, transposed), [heads * vdim, kv_rank]
        self.ff = ""                         # "", "dense", "moe"
        self.w_gu = self.w_down = None       # dense: [2 ff, width], [width, ff]; moe: [experts, 2 ff, width], [experts, width, ff]
        self.gu_interleaved = False          # gate / up rows in blocks of 64, as the gated GEMM epilogue reads them
        self.w_router = self.router_b = None


class Weights:
    def __init__(self, cfg: Config, device: torch.device, dtype: torch.dtype):
        self.cfg, self.device, self.dtype = cfg, device, dtype
        self.embed = self.embed_norm = self.final_norm = self.head = None
        self.layers: List[_Layer] = []       # one per layer; layers that share tensors are the same object
        self.tp_size, self.tp_rank = 1, 0

    def nbytes(self) -> int:
        ts = [self.embed, self.embed_norm, self.final_norm, self.head]
        for l in {id(l): l for l in self.layers}.values():
            ts += [v for v in vars(l).values() if isinstance(v, torch.Tensor)]
        return sum(t.numel() * t.element_size() for t in ts if isinstance(t, torch.Tensor))

    @classmethod
    def from_dir(cls, cfg: Config, path: Path, device: torch.device, dtype: torch.dtype) -> "Weights":
        from ..weights import _SafetensorsSource

        return cls._from_source(cfg, _SafetensorsSource(Path(path)), device, dtype)

    @classmethod
    def from_state_dict(cls, cfg: Config, sd: Dict[str, torch.Tensor], device: torch.device,
                        dtype: torch.dtype = torch.bfloat16) -> "Weights":
        from ..weights import _DictSource

        return cls._from_source(cfg, _DictSource(sd), device, dtype)

    @classmethod
    def random(cls, cfg: Config, seed: int, device: torch.device, dtype: torch.dtype = torch.bfloat16) -> "Weights":
        """Seeded random tensors generated on the device, one at a time."""
        g = torch.Generator(device=device).manual_seed(1000 * seed + 23)
        shapes = cfg.tensor_shapes()

        class _Gen:
            def has(self, name):
                return name in shapes

            def shape(self, name):
                return shapes[name]

            def full(self, name):
                sh = shapes[name]
                r = torch.randn(sh, generator=g, device=device)
                if len(sh) == 2:
                    return r * (sh[1] ** -0.5)
                if name.rsplit(".", 1)[-1] in ("b", "sink"):
                    return 0.1 * r
                return 1.0 + 0.1 * r

        return cls._from_source(cfg, _Gen(), device, dtype)

    @classmethod
    def _from_source(cls, cfg: Config, src, device: torch.device, dtype: torch.dtype) -> "Weights":
        w = cls(cfg, device, dtype)
        want = cfg.tensor_shapes()

        def get(name: str) -> torch.Tensor:
            if not src.has(name):
                raise KeyError(f"checkpoint has no tensor {name!r}")
            t = src.full(name)
            if tuple(t.shape) != tuple(want[name]):
                raise ValueError(f"{name}: shape {tuple(t.shape)}, configuration says {tuple(want[name])}")
            return t

        def dev(t: torch.Tensor) -> torch.Tensor:
            return t.to(device=device, dtype=dtype).contiguous()

        def f32(t) -> torch.Tensor:
            return torch.as_tensor(t).to(device=device, dtype=torch.float32).contiguous()

        w.embed, w.embed_norm = dev(get("embed")), dev(get("embed.norm"))
        w.final_norm, w.head = dev(get("final.norm")), dev(get("head"))
        own: Dict[int, _Layer] = {}
        for i, spec in enumerate(cfg.layers):
            if cfg.source(i) != i:
                continue
            p, m, c, l = f"l{i}.", f"l{i}.mix.", spec["mixer"], _Layer()
            l.kind = spec["type"]
            l.norm1, l.w_o = dev(get(p + "norm1")), dev(get(m + "o"))
            if l.kind == "attention":
                l.w_in = dev(torch.cat([get(m + nm) for nm in ("q", "k", "v", "g")], 0))
                l.bq, l.bk, l.bv = (dev(get(m + nm + ".b")) for nm in ("q", "k", "v"))
                l.q_norm, l.k_norm, l.sinks = dev(get(m + "q.norm")), dev(get(m + "k.norm")), f32(get(m + "sink"))
            elif l.kind == "retention":
                l.w_in = dev(torch.cat([get(m + nm) for nm in ("q", "k", "v", "g")], 0))
                l.decay = f32([float(x) for x in c["decay"]])
            else:
                H, D, C = int(c["heads"]), int(c["dim"]), int(c["kv_rank"])
                l.w_in = dev(torch.cat([get(m + "q"), get(m + "dkv")], 0))
                l.dkv_norm, l.sinks = dev(get(m + "dkv.norm")), f32(get(m + "sink"))
                l.w_ukt = dev(get(m + "uk").reshape(H, D, C).transpose(1, 2).reshape(H * C, D))
                l.w_uv = dev(get(m + "uv"))
            mlp = spec.get("mlp")
            if mlp is not None:
                f = p + "mlp."
                l.norm2 = dev(get(p + "norm2"))
                if mlp.get("kind", "dense") == "dense":
                    l.ff = "dense"
                    gu, l.gu_interleaved = gate_up_matrix(get(f + "gate"), get(f + "up"), cfg.width, dtype)
                    l.w_gu, l.w_down = dev(gu), dev(get(f + "down"))
                else:
                    l.ff = "moe"
                    l.w_router, l.router_b = dev(get(f + "router")), f32(get(f + "router.b"))
                    gus, downs = [], []
                    for e in range(int(mlp["router"]["experts"])):
                        gu, l.gu_interleaved = gate_up_matrix(get(f"{f}e{e}.gate"), get(f"{f}e{e}.up"), cfg.width, dtype)
                        gus.append(dev(gu))
                        downs.append(dev(get(f"{f}e{e}.down")))
                    l.w_gu, l.w_down = torch.stack(gus, 0).contiguous(), torch.stack(downs, 0).contiguous()
            own[i] = l
        w.layers = [own[cfg.source(i)] for i in range(len(cfg.layers))]
        return w


# ---- the layer program ------------------------------------------------------------------------------------------------


def _pad4(n: int) -> int:
    return (n + 3) // 4 * 4


class Program:
    needs_seq_view = True     # kernels walk the step sequence by sequence (ModelRunner._stage_seq)
    graph_safe = True         # a row staged without a sequence is skipped by every kernel that touches pages or state

    def __init__(self, r) -> None:
        self.r = r
        cfg: Config = r.m
        w: Weights = r.w
        e = r.e
        self.cfg, self.w = cfg, w
        if e.tp_size != 1:
            raise ValueError("Sutosun runs on one GPU per replica (no tensor-parallel split of the state mixers)")
        xt = w.dtype
        self.dt = _cabi.DT_F32 if xt == torch.float32 else _cabi.DT_BF16
        self.xt, self.esz = xt, (4 if xt == torch.float32 else 2)
        dev, T, lib = r.dev, r.Tmax, r.lib
        W, f32 = cfg.width, torch.float32
        n_q = n_lat = n_rec = n_gu = n_act = n_rl = 1
        n_in = max((l.w_in.shape[0] for l in w.layers), default=1)
        n_mix = max((l.w_o.shape[1] for l in w.layers), default=1)
        for spec in cfg.layers:
            c = spec["mixer"]
            H, D = int(c["heads"]), int(c["dim"])
            if spec["type"] == "attention":
                n_q = max(n_q, H * D)
            elif spec["type"] == "latent_attention":
                C = int(c["kv_rank"])
                n_q, n_lat = max(n_q, H * (C + int(c["rot_dim"]))), max(n_lat, H * C)
            else:
                n_rec = max(n_rec, H * int(c["vdim"]))
            mlp = spec.get("mlp")
            if mlp is None:
                continue
            if mlp.get("kind", "dense") == "dense":
                n_gu, n_act = max(n_gu, 2 * int(mlp["ff"])), max(n_act, int(mlp["ff"]))
            else:
                n_rl = max(n_rl, int(mlp["router"]["experts"]))
        if all(l.gu_interleaved for l in w.layers if l.ff == "dense"):
            n_gu = 1      # the gated epilogue writes the activation itself
        self.h = torch.zeros(T, W, dtype=f32, device=dev)          # residual stream
        # fp32 GEMM outputs of a sublayer, which one pass clears where split-K accumulates into them: the mixer's input projections;
        # then, in the same space, the feed-forward's gate / up or router outputs
        self.scratch = torch.zeros(T * max(_pad4(n_in), _pad4(n_gu), _pad4(n_rl)) + 32, dtype=f32, device=dev)
        self.rec = torch.zeros(T * n_rec, dtype=f32, device=dev)   # recurrence output
        self.xn = torch.zeros(T, W, dtype=xt, device=dev)          # the normed rows a sublayer reads
        self.q_flat = torch.zeros(T * n_q, dtype=xt, device=dev)
        self.lat_flat = torch.zeros(T * n_lat, dtype=xt, device=dev)
        self.mix_flat = torch.zeros(T * n_mix, dtype=xt, device=dev)
        self.act_flat = torch.zeros(T * n_act, dtype=xt, device=dev)
        self.xl = torch.zeros(r.Rmax, W, dtype=xt, device=dev)
        self.experts = Experts(lib, r._ck, [s["mlp"] for s in cfg.layers if (s.get("mlp") or {}).get("kind") == "moe"], T, W, self.xn,
                               self.dt, gated=True, score=_cabi.MOE_SOFTMAX, normalize=1)
        self.attention = PagedAttention(r, self.dt, max((int(s["mixer"]["heads"]) for s in cfg.layers), default=1))
        self._views: Dict[Tuple[int, int], torch.Tensor] = {}

        def view(flat: torch.Tensor, k: int) -> torch.Tensor:
            key = (flat.data_ptr(), k)
            if key not in self._views:
                self._views[key] = flat[:T * k].view(T, k)
            return self._views[key]

        # ---- linears (TMA descriptors are per (weight, input buffer) pair); layers that share tensors share them -----
        plans: Dict[int, dict] = {}
        for l in w.layers:
            if id(l) in plans:
                continue
            d = plans[id(l)] = {"in": _Linear(lib, l.w_in, self.xn, self.dt),
                                "o": _Linear(lib, l.w_o, view(self.mix_flat, l.w_o.shape[1]), self.dt)}
            if l.ff == "dense":
                d["gu"] = _Linear(lib, l.w_gu, self.xn, self.dt)
                d["down"] = _Linear(lib, l.w_down, view(self.act_flat, l.w_down.shape[1]), self.dt)
            elif l.ff == "moe":
                d["router"] = _Linear(lib, l.w_router, self.xn, self.dt)
                d["experts"] = self.experts.plans(l.w_gu, l.w_down)
        self.lin: List[dict] = [plans[id(l)] for l in w.layers]
        self.lin_head = _Linear(lib, w.head, self.xl, self.dt)
        if self.lin_head.plan is not None and cfg.logit_softcap:
            self.lin_head.plan.set_gate(1.0, cfg.logit_softcap, 0.0)   # the cap runs in the GEMM's epilogue

        # ---- pages and state slots: every layer has its own, whoever's tensors it runs -------------------------------
        bs, S = r.bs, r.Smax
        page_bytes = max(1, cfg.kv_bytes_per_token(self.esz)) * bs
        if e.num_gpu_blocks is not None:
            nb = int(e.num_gpu_blocks)
        else:
            free, total = torch.cuda.mem_get_info(dev)
            budget = int(total * e.gpu_memory_utilization) - (total - free) - (512 << 20)
            budget -= cfg.state_bytes_per_sequence() * S
            nb = min(budget // page_bytes, r.MB * S)
            if nb < r.MB:
                raise RuntimeError(f"KV budget holds {nb} blocks; one sequence of max_model_len needs {r.MB}")
        r.num_blocks = nb
        r.block_bytes = page_bytes
        self.kv: List[Optional[Tuple[torch.Tensor, torch.Tensor]]] = []   # (keys, values); a latent layer's are one array
        self.state: List[Optional[torch.Tensor]] = []
        self.rot: Dict[tuple, torch.Tensor] = {}
        self._opts: List[Optional[_cabi.AttnOpts]] = []
        for spec, l in zip(cfg.layers, w.layers):
            c = spec["mixer"]
            kv = st = o = None
            if l.kind == "retention":
                st = torch.zeros(S, int(c["heads"]), int(c["dim"]), int(c["vdim"]), dtype=f32, device=dev)
            elif l.kind == "attention":
                kv = tuple(torch.zeros(nb, int(c["kv_heads"]), bs, int(c[k]), dtype=xt, device=dev) for k in ("dim", "vdim"))
            else:
                page = torch.zeros(nb, 1, bs, int(c["kv_rank"]) + int(c["rot_dim"]), dtype=xt, device=dev)
                kv = (page, page)
            key = _rot_key(c) if l.kind != "attention" else None
            if key is not None and key not in self.rot:
                sc = dict(zip(("factor", "original", "fast", "slow"), key[2])) if key[2] else None
                freqs, mag = stretched_frequencies(key[0], key[1], sc)
                self.rot[key] = rotation_table_scaled(freqs, mag, e.max_model_len, dev)
            if kv is not None:
                o = _cabi.AttnOpts()
                o.scale, o.softcap, o.out_scale = float(c["scale"]), 0.0, 1.0
                o.chunk, o.window, o.keep_first, o.sink = 0, 0, 0, 1
                o.weight, o.gate_elem = _cabi.ATTN_SOFTMAX, 0
                o.slopes, o.sinks, o.bias = None, l.sinks.data_ptr(), None
            self.kv.append(kv)
            self.state.append(st)
            self._opts.append(o)

    def _rotation(self, c: dict) -> Tuple[Optional[int], int]:
        key = _rot_key(c)
        return (self.rot[key].data_ptr(), key[1]) if key is not None else (None, 0)

    # ------------------------------------------------------------------------------------------------------------------
    # The mixers: proj holds the layer's input projections (fp32, pitch ld), out receives the heads. Return the launch count.

    def _attention(self, li: int, proj: int, ld: int, out: int, ldo: int, T: int, n_dec: int, n_pf: int, fl: int, st: int) -> int:
        """proj columns [q | k | v | g]: biases, norms over whole projections, query factor, page write, attention."""
        r, dp = self.r, self.r._dp
        c, l = self.cfg.layers[li]["mixer"], self.w.layers[li]
        H, G, D, V = (int(c[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        o_k, o_v, o_g = H * D, (H + G) * D, (H + G) * D + G * V
        qt = c.get("q_temp") or {"coef": 0.0, "every": 1.0}
        q, (kc, vc) = self.q_flat.data_ptr(), (t.data_ptr() for t in self.kv[li])
        r._ck(r.lib.atx_qk_prepare_temp(proj, ld, 0, o_k, o_v, l.bq.data_ptr(), l.bk.data_ptr(), l.bv.data_ptr(), l.q_norm.data_ptr(),
                                        l.k_norm.data_ptr(), None, 0, float(qt["coef"]), float(qt["every"]), dp["pos"], dp["slots"],
                                        q, kc, vc, T, H, G, D, V, r.bs, self.cfg.eps, self.dt, fl, st))
        return 1 + self.attention.run(self._opts[li], q, kc, vc, D, V, H, G, D, V, proj + 4 * o_g, ld, out, ldo, T, n_dec, n_pf, fl, st)

    def _retention(self, li: int, proj: int, ld: int, out: int, ldo: int, T: int, n_dec: int, n_pf: int, fl: int, st: int) -> int:
        """proj columns [q | k | v | g]: rotation and recurrence, unit rms per head, gate. Single decoded tokens (the first n_dec
        sequences) run token by token on the FMA pipe; prompt portions in chunks on the tensor cores when the elements are bf16 and
        the kernel has the key size, else token by token as well."""
        r, lib, ck, dp = self.r, self.r.lib, self.r._ck, self.r._dp
        c, l = self.cfg.layers[li]["mixer"], self.w.layers[li]
        H, D, V = (int(c[k]) for k in ("heads", "dim", "vdim"))
        table, rd = self._rotation(c)
        rec = self.rec.data_ptr()
        args = (proj, ld, proj + 4 * H * D, ld, proj + 8 * H * D, ld, H, H, D, V, l.decay.data_ptr(), None, None, None, 0, table, rd,
                float(D) ** -0.5, self.state[li].data_ptr(), rec, H * V)
        seqs = tuple(dp[k] for k in ("seq_start", "seq_count", "seq_pos0", "seq_slot"))
        chunked = n_pf > 0 and self.xt == torch.bfloat16 and lib.atx_linear_recurrence_chunked_supported(D)
        n_seq = n_dec if chunked else n_dec + n_pf
        n = 1
        if n_seq:
            ck(lib.atx_linear_recurrence_rot(*args, *seqs, n_seq, fl, st))
            n += 1
        if chunked:
            ck(lib.atx_linear_recurrence_rot_chunked(*args, *(p + 4 * n_dec for p in seqs), n_pf, fl, st))
            n += 1
        ck(lib.atx_gated_norm_groups(rec, H * V, proj + 4 * (2 * H * D + H * V), ld, None, 0, out, ldo, T, H * V, H, self.cfg.eps, 2,
                                     1.0, self.dt, fl, st))
        return n

    def _latent(self, li: int, proj: int, ld: int, out: int, ldo: int, T: int, n_dec: int, n_pf: int, fl: int, st: int) -> int:
        """proj columns [q: per head dim plain, rot_dim rotated | latent | shared key part]."""
        r, lib, ck, dp, dt = self.r, self.r.lib, self.r._ck, self.r._dp, self.dt
        c, l = self.cfg.layers[li]["mixer"], self.w.layers[li]
        H, D, R, V, C = (int(c[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        table, rd = self._rotation(c) if R else (None, 0)
        page, qb, lat = self.kv[li][0].data_ptr(), self.q_flat.data_ptr(), self.lat_flat.data_ptr()
        seg = _cabi.HeadSeg
        # [normed latent | rotated key part] -> the token's page row; rotated query parts -> their place behind the absorbed part
        sg = [seg(src_off=H * (D + R), src_stride=C + R, heads=1, width=C + R, norm_dims=C, norm_w=l.dkv_norm.data_ptr(), rot_off=C,
                  rot_dims=rd, rot=table, rot_half=1, dst_kind=_cabi.HEAD_DST_PAGES, dst=page, dst_off=0, dst_stride=C + R)]
        if R:
            sg.append(seg(src_off=D, src_stride=D + R, heads=H, width=R, rot_off=0, rot_dims=rd, rot=table, rot_half=1,
                          dst_kind=_cabi.HEAD_DST_ROWS, dst=qb, dst_ld=H * (C + R), dst_off=C, dst_stride=C + R))
        ck(lib.atx_head_prepare(proj, ld, _cabi.head_segs(*sg), len(sg), dp["pos"], dp["slots"], T, r.bs, self.cfg.eps, dt, fl, st))
        # queries in the latent's coordinates: [W_uk,h^T q_plain | rotated q part] per head
        ck(lib.atx_head_gemm(proj, 1, ld, 0, D + R, l.w_ukt.data_ptr(), D, None, 0, qb, H * (C + R), 0, C + R, T, H, C, D, dt, fl, st))
        n = 3 + self.attention.run(self._opts[li], qb, page, page, C + R, C + R, H, 1, C + R, C, None, 0, lat, H * C, T, n_dec, n_pf,
                                   fl, st)
        ck(lib.atx_head_gemm(lat, 0, H * C, 0, C, l.w_uv.data_ptr(), C, None, 0, out, ldo, 0, V, T, H, V, C, dt, fl, st))
        return n

    def forward(self, T: int, n_dec: int, n_pf: int, n_rows: int) -> int:
        """Issue every kernel of one step on the current stream; returns the launch count. The step's first n_dec
        sequences are single decoded tokens (rows 0 .. n_dec-1), the next n_pf are prompt portions."""
        r, cfg, w, ex = self.r, self.cfg, self.w, self.experts
        lib, ck, dp, fl, dt = r.lib, r._ck, r._dp, r.flags, self.dt
        st = torch.cuda.current_stream().cuda_stream
        W, V = cfg.width, cfg.vocab_size
        h, xn, mix, act, buf = (t.data_ptr() for t in (self.h, self.xn, self.mix_flat, self.act_flat, self.scratch))
        n = 0
        probe = r.layer_probe
        small = T <= 64          # decode-sized: split-K GEMMs accumulate into buffers that the residual kernel clears
        start, pending = True, 0   # the stream does not exist yet; choices per token of expert outputs that wait to be added

        def resid(w_norm=None, out=None, rows=None, rows_n: int = T, zero_bytes: int = 0) -> None:
            """The stream starts as the normed embedding row, or takes the expert outputs that wait; its norm goes out."""
            nonlocal n, start, pending
            t = _cabi.ResidTerms()
            t.y_scale = 1.0
            if start:
                t.table_mode, t.ids, t.table, t.table_w, t.vocab = _cabi.TABLE_START, dp["ids"], w.embed.data_ptr(), w.embed_norm.data_ptr(), V
            if pending:
                t.experts, t.wgt, t.slot_of = ex.out.data_ptr(), ex.wgt.data_ptr(), ex.slot_of.data_ptr()
                t.lde, t.top = W, pending
            ck(lib.atx_parallel_resid_norm(h, ctypes.byref(t), w_norm, out, None, None, 0.0, rows, rows_n, W, cfg.eps,
                                           buf if zero_bytes else None, (zero_bytes + 15) // 16 * 16, dt, fl, st))
            n += 1
            if rows is None:
                start, pending = False, 0

        mixers = {"attention": self._attention, "retention": self._retention, "latent_attention": self._latent}
        for li, (spec, l, lin) in enumerate(zip(cfg.layers, w.layers, self.lin)):
            ld, ldo = l.w_in.shape[0], l.w_o.shape[1]
            acc = lin["in"].accumulates(T)
            resid(l.norm1.data_ptr(), xn, zero_bytes=4 * T * ld if acc else 0)
            lin["in"].run(buf, ld, T, fl, st, zeroed=acc)
            n += 2 + mixers[l.kind](li, buf, ld, mix, ldo, T, n_dec, n_pf, fl, st)
            lin["o"].run(h, W, T, fl, st, mode=_cabi.GEMM_ADD_F32)
            if l.ff == "dense":
                F = l.w_down.shape[1]
                if l.gu_interleaved:     # the gate runs in the GEMM's epilogue
                    resid(l.norm2.data_ptr(), xn)
                    lin["gu"].run(act, F, T, fl, st, mode=_cabi.GEMM_GEGLU_BF16)
                    n += 1
                else:
                    acc = lin["gu"].accumulates(T)
                    resid(l.norm2.data_ptr(), xn, zero_bytes=8 * T * F if acc else 0)
                    lin["gu"].run(buf, 2 * F, T, fl, st, zeroed=acc)
                    ck(lib.atx_gated_act_kind(buf, act, T, F, _cabi.ACT_GELU_TANH, dt, fl, st))
                    n += 2
                lin["down"].run(h, W, T, fl, st, mode=_cabi.GEMM_ADD_F32)
                n += 1
            elif l.ff == "moe":
                E, top = l.w_router.shape[0], int(spec["mlp"]["router"]["top"])
                acc = lin["router"].accumulates(T)
                resid(l.norm2.data_ptr(), xn, zero_bytes=4 * T * E if acc else 0)
                lin["router"].run(buf, E, T, fl, st, zeroed=acc)
                n += 1 + ex.run(buf, E, top, l.w_gu, l.w_down, lin["experts"], T, small, fl, st, bias=l.router_b.data_ptr())
                pending = top
            if probe is not None:
                if pending:
                    resid()
                probe.append(self.h[:T].clone())
        if n_rows:
            resid(w.final_norm.data_ptr(), self.xl.data_ptr(), rows=dp["rows"], rows_n=n_rows)
            lg, cap = r.logits.data_ptr(), cfg.logit_softcap
            if cap and self.lin_head.plan is not None:
                self.lin_head.run(lg, V, n_rows, fl, st, mode=_cabi.GEMM_SOFTCAP_F32)
            else:
                self.lin_head.run(lg, V, n_rows, fl, st)
                if cap:
                    ck(lib.atx_soft_cap(lg, V, n_rows, V, cap, fl, st))
                    n += 1
            ck(lib.atx_sample(lg, V, dp["temps"], dp["top_p"], dp["seeds"], dp["steps"], r.out_ids.data_ptr(), n_rows, V, fl, st))
            n += 2
        return n

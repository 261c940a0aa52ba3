"""Lifuzen: a decoder-only family whose layers are listed one by one in config.json, every layer PARALLEL with two norms:

    x_t = embed[token_t]
    x  <- x + m (mixer(nrm(x, w1)) + ffn(nrm(x, w2)))        nrm(x, w) = x / rms(x) * (1 + w); ffn optional
    logits = cap tanh(embed . nrm(x, w_final) / cap)

A block of consecutive layers may run several times with the same weights (`loop`); every pass has caches and states of its
own. Before a pass the stream gains the embedding output (all passes but the first) and the pass's own vector. Two mixers:

* `mamba2`: selective state-space scan: in-projection [z | x | B | C | dt], short causal convolution + silu over x, B, C,
  dt = softplus(dt + bias), S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x, gate silu(z) BEFORE an RMS norm in equal
  groups, projection.
* `attention`: soft-max attention with grouped key/value heads. The q and k projections pass a short causal convolution over
  time per channel; the values are the convolved keys as they are; then q and k are rotated (adjacent pairs, the first rot.dims
  elements of a head) and divided by their root mean square over the head. No window; 1 added to the soft-max denominator.

The feed-forward is a mixture of experts W_down max(W_up x, 0)^2: sigmoid scores, the `top` largest chosen, each chosen expert
reading its input times its score. An expert is homogeneous of degree two and the score positive, so expert(s x) = s^2 expert(x):
the products run on the plain rows and the weighted sum takes squared scores.

State besides the pages, per live sequence (a state slot): the last taps - 1 projected rows of every convolution and the
[heads, state, vdim] fp32 state of every mamba2 layer run.

fp32 whatever the element type: the residual stream, all norms, rotation, scores and weights of the attention, both
convolutions' sums, step sizes, decays, the recurrence and its state, router logits, scores and the weighted sum, the logit
cap. Projections run in the element type (bf16 on the tcgen05 GEMM and the tensor-core expert products, or fp32 on the FMA
pipe) with fp32 accumulation.

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
from .common import Experts, PagedAttention, _Linear, rotation_table

MIXERS = ("mamba2", "attention")
NORM_SHIFT = 1.0       # norm weights are stored around zero

# ---- configuration --------------------------------------------------------------------------------------------------


def _rot_key(c: dict) -> Optional[Tuple[float, int]]:
    rot = c.get("rot") or {}
    dims = int(rot.get("dims", 0) or 0)
    return (float(rot["base"]), dims) if dims else None


@dataclass
class Config:
    name: str = "lifuzen"
    vocab_size: int = 0
    width: int = 0
    eps: float = 1e-5
    residual_mult: float = 1.0
    logit_softcap: float = 0.0                         # 0: logits as they are
    layers: List[dict] = field(default_factory=list)   # {"type", "mixer", "mlp"} as in config.json
    loop: Optional[dict] = None                        # {"start", "stop", "times"}
    eos_token_ids: tuple = ()
    bos_token_id: int = 0
    max_position_embeddings: int = 131072    # the design sets no limit; this bounds the server's default max_model_len
    architecture = "Lifuzen"
    recurrent = True      # a state slot per sequence: convolution inputs, recurrent states

    @classmethod
    def from_json(cls, d: dict, name: str = "lifuzen") -> "Config":
        loop = d.get("loop") or None
        cfg = cls(name=name, vocab_size=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]),
                  residual_mult=float(d.get("residual_mult", 1.0)), logit_softcap=float(d.get("logit_softcap") or 0.0),
                  layers=[json.loads(json.dumps(l)) for l in d["layers"]],
                  loop={k: int(loop[k]) for k in ("start", "stop", "times")} if loop else None)
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.logit_softcap < 0:
            raise ValueError(f"logit_softcap={self.logit_softcap} must not be negative")
        for i, l in enumerate(self.layers):
            if l["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            c = l["mixer"] = dict(l["mixer"])
            if int(c["conv"]) < 1:
                raise ValueError(f"layer {i}: conv={c['conv']} taps")
            if l["type"] == "attention":
                c.setdefault("kv_heads", c["heads"])
                if c["heads"] % c["kv_heads"]:
                    raise ValueError(f"layer {i}: {c['heads']} heads over {c['kv_heads']} key/value heads")
                if int(c.setdefault("vdim", c["dim"])) != int(c["dim"]):
                    raise ValueError(f"layer {i}: vdim={c['vdim']} but the values are the keys (dim={c['dim']})")
                rk = _rot_key(c)
                if rk is not None and (rk[1] % 2 or rk[1] > c["dim"]):
                    raise ValueError(f"layer {i}: rot.dims={rk[1]} must be even and at most dim={c['dim']}")
            else:
                c.setdefault("groups", 1)
                c.setdefault("norm_groups", 1)
                if c["heads"] % c["groups"]:
                    raise ValueError(f"layer {i}: {c['heads']} heads over {c['groups']} groups")
                if c["heads"] * c["vdim"] % c["norm_groups"]:
                    raise ValueError(f"layer {i}: {c['heads'] * c['vdim']} channels in {c['norm_groups']} norm groups")
            mlp = l.get("mlp")
            if mlp is not None:
                if mlp.get("kind", "moe") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
                r = mlp["router"]
                if not 0 < int(r["top"]) <= int(r["experts"]):
                    raise ValueError(f"layer {i}: top={r['top']} of {r['experts']} experts")
        if self.loop:
            a, b, n = self.loop["start"], self.loop["stop"], self.loop["times"]
            if not (0 <= a < b <= len(self.layers) and n >= 1):
                raise ValueError(f"bad loop {self.loop}")

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.runs())

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer index, pass number or None) in execution order; a looped layer appears once per pass."""
        n = len(self.layers)
        if not self.loop:
            return [(i, None) for i in range(n)]
        a, b, t = self.loop["start"], self.loop["stop"], self.loop["times"]
        return ([(i, None) for i in range(a)] + [(i, p) for p in range(t) for i in range(a, b)] +
                [(i, None) for i in range(b, n)])

    def tensor_shapes(self) -> Dict[str, Tuple[int, ...]]:
        """Name -> shape of every tensor of a checkpoint of this configuration."""
        W, out = self.width, {}
        out["embed"] = (self.vocab_size, W)
        if self.loop:
            out["loop.step"] = (self.loop["times"], W)
        for i, l in enumerate(self.layers):
            p, c, m = f"l{i}.", l["mixer"], f"l{i}.mix."
            H, K = int(c["heads"]), int(c["conv"])
            out[p + "norm1"] = (W,)
            if l["type"] == "mamba2":
                P, N, G = int(c["vdim"]), int(c["state"]), int(c["groups"])
                inner, ch = H * P, H * P + 2 * G * N
                out.update({m + "in": (inner + ch + H, W), m + "conv": (ch, K), m + "conv.b": (ch,), m + "dt_bias": (H,),
                            m + "A_log": (H,), m + "D": (H,), m + "norm": (inner,), m + "o": (W, inner)})
            else:
                G, D = int(c["kv_heads"]), int(c["dim"])
                out.update({m + "q": (H * D, W), m + "k": (G * D, W), m + "q.conv": (H * D, K), m + "k.conv": (G * D, K),
                            m + "o": (W, H * D)})
            mlp = l.get("mlp")
            if mlp is not None:
                E, F, f = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"]), p + "mlp."
                out[p + "norm2"] = (W,)
                for e in range(E):
                    out[f"{f}e{e}.up"], out[f"{f}e{e}.down"] = (F, W), (W, F)
                out[f + "router"] = (E, W)
        out["final.norm"] = (W,)
        return out

    # ---- bytes, for the benchmarks' rooflines -------------------------------------------------------------------
    def weight_bytes_per_decode_step(self, elem: int = 2, tokens: int = 1) -> int:
        """Weight bytes a decode step of `tokens` tokens streams: every matrix once per run of its layer (the embedding table
        once, as the output head); of the experts at most tokens * top per layer."""
        sh = self.tensor_shapes()
        per_layer: Dict[int, int] = {}
        for k, v in sh.items():
            if k[0] == "l" and k[1].isdigit() and ".mlp.e" not in k:
                i = int(k[1:k.index(".")])
                per_layer[i] = per_layer.get(i, 0) + math.prod(v)
        n = math.prod(sh["embed"])
        for i, _ in self.runs():
            n += per_layer[i]
            mlp = self.layers[i].get("mlp")
            if mlp is not None:
                r = mlp["router"]
                n += min(int(r["experts"]), tokens * int(r["top"])) * 2 * int(mlp["expert"]["ff"]) * self.width
        return elem * n

    def kv_bytes_per_token(self, elem: int = 2) -> int:
        return sum(2 * int(self.layers[i]["mixer"]["kv_heads"]) * int(self.layers[i]["mixer"]["dim"]) * elem
                   for i, _ in self.runs() if self.layers[i]["type"] == "attention")

    def state_bytes_per_sequence(self) -> int:
        n = 0
        for i, _ in self.runs():
            c = self.layers[i]["mixer"]
            n += (int(c["conv"]) - 1) * conv_channels(self.layers[i]) * 4
            if self.layers[i]["type"] == "mamba2":
                n += int(c["heads"]) * int(c["state"]) * int(c["vdim"]) * 4
        return n

    def decode_kv_bytes(self, ctx: int, elem: int = 2) -> int:
        """Page bytes one decoded token at context length ctx reads."""
        return ctx * self.kv_bytes_per_token(elem)


def conv_channels(layer: dict) -> int:
    """Channels of a layer's short convolution: x, B and C of a mamba2 mixer, q and k of an attention mixer."""
    c = layer["mixer"]
    if layer["type"] == "mamba2":
        return int(c["heads"]) * int(c["vdim"]) + 2 * int(c["groups"]) * int(c["state"])
    return (int(c["heads"]) + int(c["kv_heads"])) * int(c["dim"])


def named_shape(name: str) -> Optional[Config]:
    """`random:lifuzen-<size>`: shapes whose layers resemble a real model's, for benchmarks (no checkpoint exists).
    `lifuzen-8b` / `lifuzen-1b` have the width, vocabulary and depth of the Llama 8B / 1B shapes; layers in the pattern
    attention, mamba2, mamba2, attention, each with 8 experts of a quarter of the feed-forward size, 2 chosen."""
    key = name.lower()
    shapes = {"lifuzen-8b": (4096, 14336, 8, 128256), "lifuzen-1b": (2048, 8192, 4, 128256),
              "lifuzen-tiny": (256, 512, 1, 1024)}     # width, feed-forward, repeats of the 4-layer pattern, vocabulary
    if key not in shapes:
        return None
    W, F, groups, vocab = shapes[key]
    hd = 128 if W >= 4096 else 64
    heads = W // hd
    moe = {"kind": "moe", "expert": {"ff": max(64, F // 4 // 64 * 64)}, "router": {"experts": 8, "top": 2}}
    att = {"type": "attention", "mlp": moe,
           "mixer": {"conv": 4, "dim": hd, "heads": heads, "kv_heads": max(1, heads // 4), "vdim": hd, "scale": hd ** -0.5,
                     "rot": {"base": 500000.0, "dims": hd // 2}}}
    mamba = {"type": "mamba2", "mlp": moe,
             "mixer": {"conv": 4, "groups": max(1, heads // 8), "heads": 2 * W // 64, "norm_groups": 1, "state": 128, "vdim": 64}}
    cfg = Config(name=key, vocab_size=vocab, width=W, eps=1e-5, residual_mult=0.7, logit_softcap=30.0,
                 layers=json.loads(json.dumps([att, mamba, mamba, att] * groups)), loop=None)
    cfg.validate()
    return cfg


# ---- weights ----------------------------------------------------------------------------------------------------------


class _Layer:
    """Device tensors of one layer in the layout the kernels read (projections that share an input are stacked)."""

    def __init__(self) -> None:
        self.kind = ""
        self.norm1 = self.norm2 = None
        self.w_in = self.w_o = None          # mamba2: [z | x | B | C | dt]; attention: [q | k]
        self.conv = self.conv_b = None       # taps over conv_channels(); bias (mamba2)
        self.dt_bias = self.a_log = self.skip = self.mix_norm = None    # mamba2
        self.w_router = self.w_up = self.w_down = None                  # [E, width], [E, ff, width], [E, width, ff]


class Weights:
    def __init__(self, cfg: Config, device: torch.device, dtype: torch.dtype):
        self.cfg, self.device, self.dtype = cfg, device, dtype
        self.embed = self.final_norm = self.loop_step = None
        self.layers: List[_Layer] = []
        self.tp_size, self.tp_rank = 1, 0

    def nbytes(self) -> int:
        ts = [self.embed, self.final_norm, self.loop_step]
        for l in self.layers:
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
        g = torch.Generator(device=device).manual_seed(1000 * seed + 19)
        shapes = cfg.tensor_shapes()

        class _Gen:
            def has(self, name):
                return name in shapes

            def shape(self, name):
                return shapes[name]

            def full(self, name):
                sh = shapes[name]
                leaf = name.rsplit(".", 1)[-1]
                r = torch.randn(sh, generator=g, device=device)
                if leaf == "conv":
                    return 0.3 * r
                if leaf == "A_log":
                    return torch.log(1.0 + 3.0 * torch.rand(sh, generator=g, device=device))
                if leaf == "dt_bias":
                    return -2.0 + r
                if leaf == "D" or name.endswith("mix.norm"):
                    return 1.0 + 0.1 * r
                if len(sh) == 2 and name != "loop.step":
                    return r * (sh[1] ** -0.5)
                return 0.1 * r

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

        def f32(t: torch.Tensor) -> torch.Tensor:
            return t.to(device=device, dtype=torch.float32).contiguous()

        w.embed, w.final_norm = dev(get("embed")), dev(get("final.norm"))
        if cfg.loop:
            w.loop_step = dev(get("loop.step"))
        for i, spec in enumerate(cfg.layers):
            p, m, l = f"l{i}.", f"l{i}.mix.", _Layer()
            l.kind = spec["type"]
            l.norm1, l.w_o = dev(get(p + "norm1")), dev(get(m + "o"))
            if l.kind == "mamba2":
                l.w_in, l.mix_norm = dev(get(m + "in")), dev(get(m + "norm"))
                l.conv, l.conv_b = dev(get(m + "conv")), dev(get(m + "conv.b"))
                l.dt_bias, l.a_log, l.skip = dev(get(m + "dt_bias")), dev(get(m + "A_log")), f32(get(m + "D"))
            else:
                l.w_in = dev(torch.cat([get(m + "q"), get(m + "k")], 0))
                l.conv = dev(torch.cat([get(m + "q.conv"), get(m + "k.conv")], 0))
            mlp = spec.get("mlp")
            if mlp is not None:
                f, E = p + "mlp.", int(mlp["router"]["experts"])
                l.norm2, l.w_router = dev(get(p + "norm2")), dev(get(f + "router"))
                l.w_up = torch.stack([dev(get(f"{f}e{e}.up")) for e in range(E)], 0).contiguous()
                l.w_down = torch.stack([dev(get(f"{f}e{e}.down")) for e in range(E)], 0).contiguous()
            w.layers.append(l)
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
            raise ValueError("Lifuzen runs on one GPU per replica (no tensor-parallel split of the state mixers)")
        xt = w.dtype
        self.dt = _cabi.DT_F32 if xt == torch.float32 else _cabi.DT_BF16
        self.xt, self.esz = xt, (4 if xt == torch.float32 else 2)
        dev, T, lib = r.dev, r.Tmax, r.lib
        W, f32 = cfg.width, torch.float32
        self.runs = cfg.runs()
        n_in = n_rec = n_mix = n_c = n_h = n_q = n_rl = 1
        for spec in cfg.layers:
            c = spec["mixer"]
            H = int(c["heads"])
            if spec["type"] == "mamba2":
                inner, ch = H * int(c["vdim"]), conv_channels(spec)
                n_in, n_rec, n_mix = max(n_in, inner + ch + H), max(n_rec, inner), max(n_mix, inner)
                n_c, n_h = max(n_c, ch), max(n_h, H)
            else:
                hd = H * int(c["dim"])
                n_in, n_q, n_mix = max(n_in, conv_channels(spec)), max(n_q, hd), max(n_mix, hd)
            if spec.get("mlp") is not None:
                n_rl = max(n_rl, int(spec["mlp"]["router"]["experts"]))
        self.h = torch.zeros(T, W, dtype=f32, device=dev)          # residual stream
        self.y = torch.zeros(T, W, dtype=f32, device=dev)          # the mixer's output
        # fp32 GEMM outputs of a layer, back to back so that one pass clears what split-K accumulates into:
        # [the mixer's input projections | router outputs]
        self.scratch = torch.zeros(T * (_pad4(n_in) + _pad4(n_rl)) + 32, dtype=f32, device=dev)
        self.rec = torch.zeros(T * n_rec, dtype=f32, device=dev)   # recurrence output
        self.xbc = torch.zeros(T * n_c, dtype=f32, device=dev)
        self.dtb = torch.zeros(2, T * n_h, dtype=f32, device=dev)  # step sizes, decays
        self.xn = torch.zeros(T, W, dtype=xt, device=dev)          # what the mixer reads
        self.xf = torch.zeros(T, W, dtype=xt, device=dev)          # what the feed-forward reads
        self.q_flat = torch.zeros(T * n_q, dtype=xt, device=dev)
        self.mix_flat = torch.zeros(T * n_mix, dtype=xt, device=dev)
        self.xl = torch.zeros(r.Rmax, W, dtype=xt, device=dev)
        # (squared scores: the weight multiplies the input of an expert of degree two)
        self.experts = Experts(lib, r._ck, [s["mlp"] for s in cfg.layers if s.get("mlp") is not None], T, W, self.xf, self.dt, power=2)
        self._views: Dict[Tuple[int, int], torch.Tensor] = {}

        def view(flat: torch.Tensor, k: int) -> torch.Tensor:
            key = (flat.data_ptr(), k)
            if key not in self._views:
                self._views[key] = flat[:T * k].view(T, k)
            return self._views[key]

        # ---- linears (TMA descriptors are per (weight, input buffer) pair) -------------------------------------------
        self.lin: List[dict] = []
        for l in w.layers:
            d = {"in": _Linear(lib, l.w_in, self.xn, self.dt),
                 "o": _Linear(lib, l.w_o, view(self.mix_flat, l.w_o.shape[1]), self.dt)}
            if l.w_up is not None:
                d["router"] = _Linear(lib, l.w_router, self.xf, self.dt)
                d["experts"] = self.experts.plans(l.w_up, l.w_down)
            self.lin.append(d)
        self.lin_head = _Linear(lib, w.embed, self.xl, self.dt)     # the output head is the embedding table
        if self.lin_head.plan is not None and cfg.logit_softcap:
            self.lin_head.plan.set_gate(1.0, cfg.logit_softcap, 0.0)   # the cap runs in the GEMM's epilogue

        # ---- pages and state slots: one set per layer RUN (a looped layer has one per pass) ------------------------
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
        self.kv: List[Optional[Tuple[torch.Tensor, torch.Tensor]]] = []   # (normed, rotated keys; convolved keys = values)
        self.state: List[Optional[torch.Tensor]] = []
        self.conv_state: List[torch.Tensor] = []
        self.rot: Dict[Tuple[float, int], torch.Tensor] = {}
        for li, _ in self.runs:
            spec, c = cfg.layers[li], cfg.layers[li]["mixer"]
            kv = st = None
            if spec["type"] == "mamba2":
                st = torch.zeros(S, int(c["heads"]), int(c["state"]), int(c["vdim"]), dtype=f32, device=dev)
            else:
                kv = tuple(torch.zeros(nb, int(c["kv_heads"]), bs, int(c["dim"]), dtype=xt, device=dev) for _ in range(2))
                key = _rot_key(c)
                if key is not None and key not in self.rot:
                    self.rot[key] = rotation_table(key[0], key[1], e.max_model_len, dev)
            self.kv.append(kv)
            self.state.append(st)
            self.conv_state.append(torch.zeros(S, max(1, int(c["conv"]) - 1), conv_channels(spec), dtype=f32, device=dev))
        # second stream for the feed-forward of decode-sized steps (see forward)
        self.overlap_ffn = True
        self.side = torch.cuda.Stream(device=dev)
        self.ev_fork, self.ev_join = torch.cuda.Event(), torch.cuda.Event()
        self.attention = PagedAttention(r, self.dt, max(int(s["mixer"]["heads"]) for s in cfg.layers))
        self._opts: List[Optional[_cabi.AttnOpts]] = []
        for spec in cfg.layers:
            o = None
            if spec["type"] == "attention":
                o = _cabi.AttnOpts()
                o.scale, o.softcap, o.out_scale = float(spec["mixer"]["scale"]), 0.0, 1.0
                o.chunk, o.window, o.keep_first, o.sink = 0, 0, 0, 1
                o.weight, o.gate_elem = _cabi.ATTN_SOFTMAX, 0
                o.slopes, o.sinks, o.bias = None, None, None
            self._opts.append(o)

    # ------------------------------------------------------------------------------------------------------------------
    def _attention(self, ri: int, li: int, proj: int, ld: int, out: int, ldo: int, T: int, n_dec: int, n_pf: int, fl: int,
                   st: int) -> int:
        """proj columns [q | k] of one layer run: convolution, rotation, norm, page write, then attention of the step's rows over
        their sequences' pages. Returns the launch count."""
        r, lib, ck, dp, dt = self.r, self.r.lib, self.r._ck, self.r._dp, self.dt
        c, l = self.cfg.layers[li]["mixer"], self.w.layers[li]
        H, G, D, K = (int(c[k]) for k in ("heads", "kv_heads", "dim", "conv"))
        C = (H + G) * D
        key = _rot_key(c)
        table, rd = (self.rot[key].data_ptr(), key[1]) if key is not None else (None, 0)
        kc, vc = (t.data_ptr() for t in self.kv[ri])
        q, cs, taps = self.q_flat.data_ptr(), self.conv_state[ri].data_ptr(), l.conv.data_ptr()
        seg = _cabi.ConvHeadSeg
        segs = _cabi.conv_head_segs(
            seg(src_off=0, heads=H, width=D, norm=1, rot_dims=rd, dst_kind=_cabi.HEAD_DST_ROWS, w=taps, rot=table, dst=q, dst_ld=H * D),
            seg(src_off=H * D, heads=G, width=D, norm=1, rot_dims=rd, dst_kind=_cabi.HEAD_DST_PAGES, w=taps + H * D * K * self.esz,
                rot=table, dst=kc, raw_dst=vc))
        ck(lib.atx_conv_head_prepare(proj, ld, segs, 2, K, cs, C, n_dec, dp["pos"], dp["slots"], dp["tok_seq"], dp["seq_start"],
                                     dp["seq_pos0"], dp["seq_slot"], T, r.bs, self.cfg.eps, dt, fl, st))
        n = 1
        if n_pf and K > 1:
            ck(lib.atx_conv_state_update(proj, ld, 0, cs, *(dp[k] + 4 * n_dec for k in ("seq_start", "seq_count", "seq_pos0", "seq_slot")),
                                         n_pf, C, K, fl, st))
            n += 1
        return n + self.attention.run(self._opts[li], q, kc, vc, D, D, H, G, D, D, None, 0, out, ldo, T, n_dec, n_pf, fl, st)

    def _mamba2(self, ri: int, li: int, proj: int, ld: int, out: int, ldo: int, T: int, n_dec: int, n_pf: int, fl: int,
                st: int) -> int:
        """proj columns [z | x | B | C | dt] of one layer run: convolution and step sizes, scan, gated norm. Single decoded tokens
        (the first n_dec sequences) run token by token on the FMA pipe; prompt portions in chunks on the tensor cores when the
        elements are bf16 and the kernel has the state size, else token by token as well. Returns the launch count."""
        lib, ck, dp, dt = self.r.lib, self.r._ck, self.r._dp, self.dt
        c, l = self.cfg.layers[li]["mixer"], self.w.layers[li]
        H, P, N, G, K = (int(c[k]) for k in ("heads", "vdim", "state", "groups", "conv"))
        inner, ch = H * P, H * P + 2 * G * N
        seqs = (dp["seq_start"], dp["seq_count"], dp["seq_pos0"], dp["seq_slot"])
        pf_seqs = tuple(p + 4 * n_dec for p in seqs)
        xbc, dts, dec, rec, cs = (t.data_ptr() for t in (self.xbc, self.dtb[0], self.dtb[1], self.rec, self.conv_state[ri]))
        ck(lib.atx_conv_dt_inplace(proj, ld, inner, inner + ch, l.conv.data_ptr(), l.conv_b.data_ptr(), l.dt_bias.data_ptr(),
                                   l.a_log.data_ptr(), cs, xbc, dts, dec, dp["tok_seq"], dp["seq_start"], dp["seq_pos0"],
                                   dp["seq_slot"], n_dec, T, ch, H, K, dt, fl, st))
        n = 1
        if n_pf and K > 1:
            ck(lib.atx_conv_state_update(proj, ld, inner, cs, *pf_seqs, n_pf, ch, K, fl, st))
            n += 1
        args = (xbc + 4 * (inner + G * N), ch, xbc + 4 * inner, ch, xbc, ch, H, G, N, P, None, dec, dts, l.skip.data_ptr(), 0,
                self.state[ri].data_ptr(), rec, inner)
        chunked = n_pf > 0 and self.xt == torch.bfloat16 and lib.atx_linear_recurrence_chunked_supported(N)
        n_seq = n_dec if chunked else n_dec + n_pf
        if n_seq:
            ck(lib.atx_linear_recurrence(*args, *seqs, n_seq, fl, st))
            n += 1
        if chunked:
            ck(lib.atx_linear_recurrence_chunked(*args, *pf_seqs, n_pf, fl, st))
            n += 1
        ck(lib.atx_gated_norm(rec, inner, proj, ld, l.mix_norm.data_ptr(), out, ldo, T, inner, int(c["norm_groups"]), self.cfg.eps,
                              1, 1.0, dt, fl, st))
        return n + 1

    def forward(self, T: int, n_dec: int, n_pf: int, n_rows: int) -> int:
        """Issue every kernel of one step on the current stream; returns the launch count. The step's first n_dec
        sequences are single decoded tokens (rows 0 .. n_dec-1), the next n_pf are prompt portions."""
        r, cfg, w, ex = self.r, self.cfg, self.w, self.experts
        lib, ck, dp, fl, dt = r.lib, r._ck, r._dp, r.flags, self.dt
        main = torch.cuda.current_stream()
        st = main.cuda_stream
        W, V = cfg.width, cfg.vocab_size
        h, y, xn, xf, mix, proj = (t.data_ptr() for t in (self.h, self.y, self.xn, self.xf, self.mix_flat, self.scratch))
        n = 0
        probe = r.layer_probe
        small = T <= 64    # decode-sized: split-K GEMMs accumulate into buffers that the residual kernel hands back cleared
        if small:
            self.y[:T].zero_()
        pending = 0        # what the last layer left to add: 0 nothing, 1 the mixer's output, 2 that and the experts'
        pending_top = 0

        def resid(w_a=None, out_a=None, w_b=None, out_b=None, table_mode: int = 0, vec=None, rows=None, rows_n: int = T,
                  zero_bytes: int = 0) -> None:
            """The stream takes what the last layer left (and an embedding row, a pass vector); one or two norms of it go out."""
            nonlocal n, pending
            t = _cabi.ResidTerms()
            t.y_scale, t.table_mode, t.vocab = cfg.residual_mult, table_mode, V
            t.ids, t.table, t.vec = dp["ids"], w.embed.data_ptr(), vec
            if pending:
                t.y, t.zero_y = y, 1 if (small and rows is None) else 0
            if pending == 2:
                t.experts, t.wgt, t.slot_of = ex.out.data_ptr(), ex.wgt.data_ptr(), ex.slot_of.data_ptr()
                t.lde, t.top = W, pending_top
            ck(lib.atx_parallel_resid_norm(h, ctypes.byref(t), w_a, out_a, w_b, out_b, NORM_SHIFT, rows, rows_n, W, cfg.eps,
                                           proj if zero_bytes else None, zero_bytes, dt, fl, st))
            n += 1
            if rows is None:
                pending = 0

        table_mode = _cabi.TABLE_START
        for ri, (li, p) in enumerate(self.runs):
            l, lin = w.layers[li], self.lin[li]
            vec = None
            if p is not None and li == cfg.loop["start"]:      # a pass of the looped block begins
                vec = w.loop_step.data_ptr() + p * W * self.esz
                if p > 0:
                    table_mode = _cabi.TABLE_ADD
            ld, E = l.w_in.shape[0], l.w_router.shape[0] if l.w_router is not None else 0
            rl = proj + 4 * _pad4(T * ld)
            acc = lin["in"].accumulates(T)
            resid(l.norm1.data_ptr(), xn, l.norm2.data_ptr() if E else None, xf if E else None, table_mode=table_mode, vec=vec,
                  zero_bytes=(rl + 4 * T * E - proj + 15) // 16 * 16 if acc else 0)
            table_mode = 0
            # Decode-sized steps: the feed-forward does not wait for the mixer (each reads its own norm of the stream), so router,
            # plan and expert products run on a second stream beside the mixer's chain of short kernels; the streams join in
            # front of the next residual kernel. Inside a captured graph these are two branches of the layer.
            fs, side = st, None
            if E and small and self.overlap_ffn:
                side = self.side
                self.ev_fork.record(main)
                side.wait_event(self.ev_fork)
                fs = side.cuda_stream
            top = 0
            if E:
                top = int(cfg.layers[li]["mlp"]["router"]["top"])
                lin["router"].run(rl, E, T, fl, fs, zeroed=acc)
                n += 1 + ex.run(rl, E, top, l.w_up, l.w_down, lin["experts"], T, small, fl, fs)
                if side is not None:
                    self.ev_join.record(side)
            lin["in"].run(proj, ld, T, fl, st, zeroed=acc)
            K_o = l.w_o.shape[1]
            mixer = self._mamba2 if l.kind == "mamba2" else self._attention
            n += 2 + mixer(ri, li, proj, ld, mix, K_o, T, n_dec, n_pf, fl, st)
            lin["o"].run(y, W, T, fl, st, zeroed=small)
            if side is not None:
                main.wait_event(self.ev_join)
            pending, pending_top = (2, top) if E else (1, 0)
            if probe is not None:
                resid()
                probe.append(self.h[:T].clone())
        if n_rows:
            resid(w.final_norm.data_ptr(), self.xl.data_ptr(), table_mode=table_mode, rows=dp["rows"], rows_n=n_rows)
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

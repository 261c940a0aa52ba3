"""What the layer programs of the layer-list families share: the linear layer that picks a GEMM kernel, the table of
rotation angles, attention of a step's rows over their pages, the experts of a mixture."""
from __future__ import annotations

import ctypes
import math
from typing import List, Optional

import torch

from .. import _cabi


def _use_tc(dtype: torch.dtype, k: int) -> bool:
    return dtype == torch.bfloat16 and k % 64 == 0


class _Linear:
    """out[t, :] = X[t, :] @ W^T (fp32 out): the tcgen05 GEMM when the operands are bf16 and K is a multiple of its
    64-element block, else the FMA-pipe GEMM (fp32 operands, odd reduction sizes)."""

    def __init__(self, lib, w: torch.Tensor, x_buf: torch.Tensor, dt: int):
        self.lib, self.w, self.x, self.dt = lib, w, x_buf, dt
        self.N, self.K = int(w.shape[0]), int(w.shape[1])
        assert x_buf.shape[1] == self.K and x_buf.is_contiguous() and w.is_contiguous()
        self.plan = _cabi.GemmPlan(w, x_buf) if _use_tc(w.dtype, self.K) else None

    def accumulates(self, T: int) -> bool:
        """Decode-sized steps stream the weights once: the tcgen05 GEMM then cuts K over enough CTAs to fill the GPU
        and ADDS its partial sums, so the target has to be zero before the launch."""
        return self.plan is not None and T <= 64

    def run(self, out_ptr: int, ldo: int, T: int, flags: int, st: int, mode: int = _cabi.GEMM_STORE_F32,
            zeroed: bool = False) -> None:
        if self.plan is not None:
            if zeroed and mode == _cabi.GEMM_STORE_F32 and self.accumulates(T):
                rc = self.lib.atx_gemm_run(self.plan._h, out_ptr, ldo, T, _cabi.GEMM_ADD_F32, 0, flags, st)
            else:
                whole_k = mode in (_cabi.GEMM_STORE_F32, _cabi.GEMM_SOFTCAP_F32)
                rc = self.lib.atx_gemm_run(self.plan._h, out_ptr, ldo, T, mode, 1 if whole_k else 0, flags, st)
        else:
            assert mode in (_cabi.GEMM_STORE_F32, _cabi.GEMM_ADD_F32)
            rc = self.lib.atx_gemm_simple(self.w.data_ptr(), self.K, self.x.data_ptr(), self.K, out_ptr, ldo, T, self.N,
                                          self.K, 1 if mode == _cabi.GEMM_ADD_F32 else 0, self.dt, flags, st)
        if rc != 0:
            raise _cabi.AtxError(f"atx error {rc}: {self.lib.atx_last_error().decode()}")


def rotation_table(base: float, dims: int, max_pos: int, device: torch.device) -> torch.Tensor:
    """[max_pos, dims] fp32: cos then sin of p * base^(-2i/dims), i < dims/2, evaluated in float64 on the host."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    ang = torch.arange(max_pos, dtype=torch.float64)[:, None] * torch.pow(torch.tensor(base, dtype=torch.float64),
                                                                          -2.0 * i / dims)[None, :]
    return torch.cat((ang.cos(), ang.sin()), -1).to(torch.float32).contiguous().to(device)


def wavelength_scaled_frequencies(base: float, dims: int, scaling: Optional[dict]) -> List[float]:
    """f_i = base^(-2i/dims), i < dims/2, rescaled by wavelength l = 2 pi / f (`scaling` = factor, low, high, original; None:
    as they are): f stays where l < original / high, becomes f / factor where l > original / low, and between the two is
    (1 - s) f / factor + s f with s = (original / l - low) / (high - low). Float64 on the host."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            factor, low, high, orig = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
            wl = 2.0 * math.pi / f
            if wl > orig / low:
                f = f / factor
            elif wl >= orig / high:
                s = (orig / wl - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotation_table_for(freqs: List[float], max_pos: int, device: torch.device) -> torch.Tensor:
    """[max_pos, 2 * len(freqs)] fp32: cos then sin of p * f_i for the given frequencies, evaluated in float64 on the host."""
    ang = torch.arange(max_pos, dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)[None, :]
    return torch.cat((ang.cos(), ang.sin()), -1).to(torch.float32).contiguous().to(device)


def stretched_frequencies(base: float, dims: int, scaling: Optional[dict]) -> "tuple[List[float], float]":
    """f_i = base^(-2i/dims), i < dims/2, stretched by pair index (`scaling` = factor, original, fast, slow; None: as they
    are), and the magnitude that multiplies every cosine and sine. A pair that makes t turns over `original` positions has
    the index d(t) = dims ln(original / (2 pi t)) / (2 ln base); with lo = floor(d(fast)) and hi = ceil(d(slow)), clipped to
    [0, dims - 1], the share s_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1) of f_i is divided by factor:
    f_i (1 - s_i) + f_i s_i / factor. Magnitude 0.1 ln(factor) + 1. Float64 on the host."""
    freqs = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return freqs, 1.0
    factor, orig = float(scaling["factor"]), float(scaling["original"])

    def index_of(turns: float) -> float:
        return dims * math.log(orig / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))

    lo = max(math.floor(index_of(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index_of(float(scaling["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        s = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * s + f * (1.0 - s))
    return out, 0.1 * math.log(factor) + 1.0


def rotation_table_scaled(freqs: List[float], magnitude: float, max_pos: int, device: torch.device) -> torch.Tensor:
    """rotation_table_for with every cosine and sine multiplied by `magnitude` (the rotation kernels apply the table's
    entries as they are, so a rotated pair comes out scaled)."""
    ang = torch.arange(max_pos, dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)[None, :]
    return (torch.cat((ang.cos(), ang.sin()), -1) * magnitude).to(torch.float32).contiguous().to(device)


def gate_up_matrix(gate: torch.Tensor, up: torch.Tensor, width: int, dtype: torch.dtype) -> "tuple[torch.Tensor, bool]":
    """Gate and up rows as one matrix: in blocks of 64 where a gated GEMM epilogue reads them (True), else one after the other."""
    if _use_tc(dtype, width) and gate.shape[0] % 64 == 0:
        from ..weights import interleave_gate_up

        return interleave_gate_up(gate, up), True
    return torch.cat([gate, up], 0), False


class PagedAttention:
    """Attention of a step's rows over their sequences' pages: prompt portions on the tensor cores where the element type and the
    sizes have such a kernel; single decoded tokens (and every row otherwise) on the decode form of that kernel or on the kernel
    that gives a warp to each (row, head). One object serves every layer of a program."""

    def __init__(self, r, dt: int, max_heads: int):
        self.r, self.dt = r, dt
        # scratch of the decode form's key slices: [tokens, heads, slices, value width + 2] fp32
        self.max_splits = 32
        self.sms = torch.cuda.get_device_properties(r.dev).multi_processor_count
        self.ws = torch.zeros(max(2, r.Smax * max_heads * self.max_splits * (128 + 2)), dtype=torch.float32, device=r.dev)

    def run(self, opts: "_cabi.AttnOpts", q: int, kc: int, vc: int, k_row: int, v_row: int, H: int, G: int, D: int, Vd: int,
            gate: Optional[int], ldg: int, out: int, ldo: int, T: int, n_dec: int, n_pf: int, fl: int, st: int) -> int:
        """Rows 0 .. n_dec - 1 are single decoded tokens, the rest the n_pf prompt portions; a token's key row holds k_row elements
        (the key its first D), its value row v_row (the value its first Vd). Returns the launch count."""
        r, lib, ck, dp, dt = self.r, self.r.lib, self.r._ck, self.r._dp, self.dt
        po = ctypes.byref(opts)
        tc = n_pf > 0 and lib.atx_attn_window_prefill_supported(D, Vd, k_row, v_row, dt)
        rows = n_dec if tc else T
        n = 0
        if rows and rows == n_dec and lib.atx_attn_window_decode_supported(H, G, D, Vd, k_row, v_row, dt):
            # as many slices of the keys as fill the GPU about three times, by the longest span a query of this layer can see: a
            # fixed number per layer and batch size, so a captured graph stays valid
            keys = min((opts.window + opts.keep_first) if opts.window else r.e.max_model_len, r.e.max_model_len)
            splits = max(1, min((keys + 63) // 64, self.max_splits, -(-3 * self.sms // (rows * G))))
            ck(lib.atx_attn_paged_decode(q, kc, vc, k_row, v_row, dp["seq_bt"], r.MB, dp["tok_seq"], dp["pos"], gate, ldg, out, ldo,
                                         self.ws.data_ptr(), self.ws.numel() * 4, splits, rows, H, G, D, Vd, r.bs, po, dt, fl, st))
            n += 2 if splits > 1 else 1
        elif rows:
            ck(lib.atx_attn_paged(q, kc, vc, k_row, v_row, dp["seq_bt"], r.MB, dp["tok_seq"], dp["pos"], gate, ldg, out, ldo, rows,
                                  H, G, D, Vd, r.bs, po, dt, fl, st))
            n += 1
        if tc:
            # rows of the prompt portions start at row n_dec: q, gate and out are passed whole, rows come from seq_start
            ck(lib.atx_attn_paged_prefill(q, kc, vc, k_row, v_row, dp["seq_bt"] + 4 * n_dec * r.MB, r.MB,
                                          *(dp[k] + 4 * n_dec for k in ("seq_start", "seq_count", "seq_pos0")), n_pf, T - n_dec,
                                          gate, ldg, out, ldo, H, G, D, Vd, r.bs, po, dt, fl, st))
            n += 1
        return n


class Experts:
    """The feed-forwards of a mixture of experts, sum_k w_k W_down,e act_e(x): routing, the plan that sorts (token, choice) pairs by
    expert, the two products. The weighted sum is left to the kernel that consumes `out` by slot (`slot_of`, `wgt`). One object
    serves every layer of a program (its buffers are reused from layer to layer).

    gated: act = silu(W_gate x) * (W_up x), w_up holding gate and up rows (gate_up_matrix); else max(W_up x, 0)^2. score, normalize,
    power: how router outputs become weights (atx_moe_route_scored)."""

    def __init__(self, lib, ck, specs: List[dict], T: int, W: int, xn: torch.Tensor, dt: int, gated: bool = False,
                 score: int = _cabi.MOE_SIGMOID, normalize: int = 0, power: int = 1):
        """specs: the `mlp` entries of the model's layers (may be empty); xn [T, W]: the rows the experts read."""
        dev, xt, i32 = xn.device, xn.dtype, torch.int32
        self.lib, self.ck, self.W, self.dt, self.xn = lib, ck, W, dt, xn
        self.gated, self.score, self.normalize, self.power = gated, score, normalize, power
        top = max([int(m["router"]["top"]) for m in specs], default=1)
        E = max([int(m["router"]["experts"]) for m in specs], default=1)
        F = max([int(m["expert"]["ff"]) for m in specs], default=1)
        P = T * top if specs else 1
        self.P = P
        self.tile_rows, self.big_rows = int(lib.atx_moe_tile_rows()), int(lib.atx_gemm_grouped_tile_rows())
        self.max_tiles = (P + self.tile_rows - 1) // self.tile_rows + E
        self.max_big_tiles = (P + self.big_rows - 1) // self.big_rows + E
        self.sel = torch.zeros(P, dtype=i32, device=dev)
        self.wgt = torch.zeros(P, dtype=torch.float32, device=dev)
        self.seg_off = torch.zeros(E + 1, dtype=i32, device=dev)
        self.perm = torch.zeros(P, dtype=i32, device=dev)
        self.slot_of = torch.zeros(P, dtype=i32, device=dev)
        self.tiles = torch.zeros(2 + 2 * self.max_tiles, dtype=i32, device=dev)
        self.tiles_big = torch.zeros(2 + 2 * self.max_big_tiles, dtype=i32, device=dev)
        self.act = torch.zeros(P * F, dtype=xt, device=dev)
        self.out = torch.zeros(P * W if specs else 1, dtype=torch.float32, device=dev)
        self.grouped = any(_use_tc(xt, W) and int(m["expert"]["ff"]) % 64 == 0 for m in specs)
        self.xperm = torch.zeros(P if self.grouped else 1, W, dtype=xt, device=dev)

    def plans(self, w_up: torch.Tensor, w_down: torch.Tensor) -> Optional[dict]:
        """GEMM plans of one layer (w_up [E, F, W], or [E, 2 F, W] with gates; w_down [E, W, F]; the up product over gathered rows,
        and over the step's tokens as they are), or None where the sizes have none."""
        (E, N, W), F = w_up.shape, w_down.shape[2]
        if not (_use_tc(w_up.dtype, W) and F % 64 == 0):
            return None
        return {"up": _cabi.GemmPlan(w_up.view(E * N, W), self.xperm), "up_tokens": _cabi.GemmPlan(w_up.view(E * N, W), self.xn),
                "down": _cabi.GemmPlan(w_down.view(E * W, F), self.act[:self.P * F].view(self.P, F))}

    def run(self, logits: int, ld: int, top: int, w_up: torch.Tensor, w_down: torch.Tensor, plans: Optional[dict], T: int,
            small: bool, fl: int, st: int, bias: Optional[int] = None) -> int:
        """Router logits (device pointer, fp32 [T, ld]; bias [E] fp32 is added to them) -> sel, wgt, slot_of and `out` by slot.
        Returns the launch count."""
        lib, ck, W, dt = self.lib, self.ck, self.W, self.dt
        E, N, F = int(w_up.shape[0]), int(w_up.shape[1]), int(w_down.shape[2])
        sel, so, pm, sl = (t.data_ptr() for t in (self.sel, self.seg_off, self.perm, self.slot_of))
        pairs, act, out, x = T * top, self.act.data_ptr(), self.out.data_ptr(), self.xn.data_ptr()
        route = (logits, ld, bias, None, E, top, 1.0, self.normalize, self.score, self.power)
        up_mode = _cabi.GEMM_SWIGLU_BF16 if self.gated else _cabi.GEMM_RELU2_BF16
        wgt = self.wgt.data_ptr()
        if small:
            # decode-sized: one tile per chosen expert. With plans both products stream the chosen matrices on the tcgen05 kernel, the
            # first one over the step's tokens as they are; without, 64-slot tiles on the expert kernel.
            tiles, tl = min(E, pairs), self.tiles.data_ptr()
            ck(lib.atx_moe_route_plan_biased(*route, T, E, self.tile_rows, sel, wgt, so, pm, sl, tl, fl, st))
            n = 1
            if plans is not None:
                ck(lib.atx_gemm_run_grouped_small(plans["up_tokens"]._h, act, F, N, up_mode, so, tl, tiles, pm, top, T, fl, st))
                ck(lib.atx_gemm_run_grouped_small(plans["down"]._h, out, W, W, _cabi.GEMM_STORE_F32, so, tl, tiles, None, top, T, fl, st))
                return n + 2
        else:
            ck(lib.atx_moe_route_biased(*route, sel, wgt, T, fl, st))
            n = 2
            if plans is not None:
                # prompt-sized: gather every expert's rows, then both products on the persistent tcgen05 GEMM over the plan's tiles
                big, tb = min(self.max_big_tiles, (pairs + self.big_rows - 1) // self.big_rows + E), self.tiles_big.data_ptr()
                ck(lib.atx_moe_plan(sel, pairs, E, self.big_rows, so, pm, sl, tb, fl, st))
                ck(lib.atx_moe_gather_rows(x, W, pm, top, so, E, self.xperm.data_ptr(), W, pairs, W, dt, fl, st))
                ck(lib.atx_gemm_run_grouped(plans["up"]._h, act, F, N, up_mode, so, tb, big, fl, st))
                ck(lib.atx_gemm_run_grouped(plans["down"]._h, out, W, W, _cabi.GEMM_STORE_F32, so, tb, big, fl, st))
                return n + 3
            tiles, tl = min(self.max_tiles, (pairs + self.tile_rows - 1) // self.tile_rows + E), self.tiles.data_ptr()
            ck(lib.atx_moe_plan(sel, pairs, E, self.tile_rows, so, pm, sl, tl, fl, st))
        ck(lib.atx_moe_expert_gemm(x, W, pm, top, 1, w_up.data_ptr(), N * W, W, act, F, F, W, 1 if self.gated else _cabi.MOE_ACT_RELU2,
                                   1 if (self.gated and plans is not None) else 0, self.tile_rows, so, tl, tiles, dt, fl, st))
        ck(lib.atx_moe_expert_gemm(act, F, None, top, 0, w_down.data_ptr(), W * F, F, out, W, W, F, 0, 0, self.tile_rows, so, tl, tiles,
                                   dt, fl, st))
        return n + 2

"""The Lifuzen family on the GPU against the float64 reference (oracle/lifuzen_ref.py): the engine (scheduler, pages, state slots,
runner, kernels) on small random models (whole prompts, token-by-token decoding, portions down to two tokens, mixed batches,
reuse of pages and slots, greedy generation through the ordinary entry point) and kernels alone on inputs built so that a lost
state, a far key, a sink that is left out, a convolution that forgets its predecessors or a wrong expert weight shows."""
import ctypes

import numpy as np
import pytest
import torch

from oracle import lifuzen_ref as R

pytestmark = pytest.mark.gpu
F64 = torch.float64
DEV = "cuda:0"


# ---- small models ------------------------------------------------------------------------------------------------------

def moe(experts=5, top=2, ff=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def att(heads=4, kv=2, dim=12, dims=8, base=100.0, scale=0.3, conv=4, mlp=None):
    c = {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv, "vdim": dim, "scale": scale}
    if dims:
        c["rot"] = {"base": base, "dims": dims}
    return {"type": "attention", "mixer": c, "mlp": mlp}


def mamba(heads=4, vdim=10, state=6, groups=2, norm_groups=1, conv=3, mlp=None):
    return {"type": "mamba2", "mlp": mlp,
            "mixer": {"conv": conv, "groups": groups, "heads": heads, "norm_groups": norm_groups, "state": state, "vdim": vdim}}


def model_cfg(layers, width=64, vocab=96, loop=None, mult=0.6, cap=15.0, eps=1e-5):
    return {"architecture": "Lifuzen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "logit_softcap": cap, "loop": None if loop is None else dict(zip(("start", "stop", "times"), loop)), "layers": layers}


def mixed_model(width=64):
    """Both mixers, layers with and without experts, a block of three layers that runs twice between layers that run once."""
    return model_cfg([mamba(mlp=moe()), att(mlp=moe(4, 1, 40)), mamba(heads=3, vdim=8, state=5, groups=1, norm_groups=2, conv=4),
                      att(heads=6, kv=3, dim=8, dims=4, conv=2, mlp=moe(7, 3, 16)), mamba(conv=2, norm_groups=4, mlp=moe(3, 3, 8))],
                     width=width, loop=(1, 4, 2))


def engine(cfg, wt, dtype="float32", **kw):
    from atx.config import EngineConfig, ModelSource
    from atx.engine import LLMEngine
    from atx.models import lifuzen

    mcfg = lifuzen.Config.from_json(cfg)
    xt = torch.float32 if dtype == "float32" else torch.bfloat16
    w = lifuzen.Weights.from_state_dict(mcfg, wt, torch.device(DEV), xt)
    ecfg = EngineConfig(max_model_len=kw.pop("max_model_len", 256), max_num_seqs=kw.pop("max_num_seqs", 4),
                        max_num_batched_tokens=kw.pop("max_num_batched_tokens", 256),
                        num_gpu_blocks=kw.pop("num_gpu_blocks", 64),
                        enable_prefix_caching=False,
                        enable_cuda_graphs=kw.pop("enable_cuda_graphs", False),
                        async_scheduling=kw.pop("async_scheduling", False), dtype=dtype,
                        max_logit_rows=kw.pop("max_logit_rows", 256), **kw)
    return LLMEngine(ModelSource(mcfg, None, None), ecfg, w)


def tokens(n, vocab=96, seed=0):
    return [int(t) for t in torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed))]


def rel_rows(got, want):
    """Per row: rms(got - want) / rms(want), both with the row mean taken off."""
    got, want = torch.as_tensor(got, dtype=F64), torch.as_tensor(want, dtype=F64)
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt()


def rel(got, want):
    return float(rel_rows(got, want).max())


TOL = {"float32": 4e-5, "bfloat16": 0.08}      # bf16: operand rounding through the layers; fp32 is the sharp test


def chooses(cfg):
    """Some layer leaves experts out: a choice that rounding can flip."""
    return any(l.get("mlp") and l["mlp"]["router"]["top"] < l["mlp"]["router"]["experts"] for l in cfg["layers"])


def close(got, want, dtype, cfg):
    """Every row within the tolerance. One exception: a bf16 model that chooses experts. The choice is a discontinuous step, so
    where two scores of the reference lie closer than bf16 rounding of the router's input moves them the engine may rightly
    pick the other expert, and that token (and, through the mixers, later ones) then differs visibly. Random test weights have
    such close calls; there four rows in five must be within the tolerance and none may be far off. The fp32 runs of the same
    models are held to the sharp limit on every row."""
    rows = rel_rows(got, want)
    if dtype == "bfloat16" and chooses(cfg):
        return float(rows.quantile(0.8)) < TOL[dtype] and float(rows.max()) < 0.7
    return float(rows.max()) < TOL[dtype]


def whole(eng, rid, toks, end=True):
    return eng.feed([(rid, toks, list(range(len(toks))))], [rid] if end else [])


def portions(eng, rid, toks, cuts):
    parts, at = [], 0
    for n in cuts:
        parts.append(eng.feed([(rid, toks[at:at + n], list(range(n)))], [rid] if at + n == len(toks) else []))
        at += n
    assert at == len(toks)
    return np.concatenate(parts)


def run_steps(eng, reqs, steps):
    """steps: lists of (request, token count); returns the logits of every request in order of its tokens."""
    at = {k: 0 for k in reqs}
    got = {k: [] for k in reqs}
    for step in steps:
        entries, end = [], []
        for k, n in step:
            entries.append((k, reqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
            if at[k] == len(reqs[k]):
                end.append(k)
        out, o = eng.feed(entries, end), 0
        for k, n in step:
            got[k].append(out[o:o + n])
            o += n
    assert at == {k: len(v) for k, v in reqs.items()}
    return {k: np.concatenate(v) for k, v in got.items()}


# ---- each mechanism alone, through the engine ------------------------------------------------------------------------------

ONE_LAYER = {
    "attention": lambda: att(),
    "attention_no_rotation": lambda: att(dims=0),
    "attention_whole_head_turns": lambda: att(dims=12, base=30000.0),
    "attention_a_kv_head_per_query_head": lambda: att(heads=3, kv=3),
    "attention_one_head_of_two": lambda: att(heads=1, kv=1, dim=2, dims=2),
    "attention_wide_heads": lambda: att(heads=2, kv=1, dim=160, dims=64, scale=0.05),
    "attention_wider_than_the_register_path": lambda: att(heads=2, kv=1, dim=264, dims=16, scale=0.04),
    "attention_odd_head": lambda: att(heads=2, kv=1, dim=7, dims=6),
    "mamba2": lambda: mamba(),
    "mamba2_one_head": lambda: mamba(heads=1, vdim=3, state=2, groups=1),
    "mamba2_a_group_per_head": lambda: mamba(heads=4, groups=4, norm_groups=8),
    "mamba2_packed_path": lambda: mamba(heads=2, vdim=40, state=32, groups=1, norm_groups=2),
    "mamba2_wide_state": lambda: mamba(heads=2, vdim=8, state=72),
    "experts": lambda: att(mlp=moe()),
    "experts_one_of_many": lambda: mamba(mlp=moe(40, 1, 8)),
    "experts_every_one": lambda: att(mlp=moe(3, 3, 17)),
    "experts_single": lambda: mamba(mlp=moe(1, 1, 40)),
    "tensor_core_attention": lambda: att(heads=4, kv=2, dim=64, dims=32, scale=0.125, mlp=moe(4, 2, 64)),
    "tensor_core_attention_between_widths": lambda: att(heads=4, kv=1, dim=40, dims=24, scale=0.2, mlp=moe(4, 4, 128)),
    "tensor_core_scan": lambda: mamba(heads=4, vdim=48, state=64, groups=2, norm_groups=2, conv=4, mlp=moe(2, 2, 64)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [64, 88])       # 88: not a multiple of the tensor-core GEMM's K block
@pytest.mark.parametrize("kind", sorted(ONE_LAYER))
def test_one_layer_models(kind, width, dtype):
    cfg = model_cfg([ONE_LAYER[kind]()], width=width)
    wt = R.random_checkpoint(cfg, 11)
    toks = tokens(150, seed=1)
    eng = engine(cfg, wt, dtype)
    want = R.forward(cfg, wt, toks)
    got = whole(eng, "a", toks)
    assert close(got, want, dtype, cfg), (kind, width, dtype, rel(got, want))
    got = portions(eng, "b", toks, [2, 61, 1, 1, 70, 2, 13])
    assert close(got, want, dtype, cfg), (kind, width, dtype, rel(got, want))
    eng.runner.close()


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 8, 11])
def test_convolution_lengths_with_steps_shorter_than_the_taps(taps):
    cfg = model_cfg([mamba(conv=taps), att(conv=taps, dim=8, dims=4), att(heads=3, kv=3, dim=7, dims=2, conv=taps)])
    wt = R.random_checkpoint(cfg, 4)
    toks = tokens(40, seed=taps)
    want = R.forward(cfg, wt, toks)
    eng = engine(cfg, wt)
    assert rel(whole(eng, "w", toks), want) < TOL["float32"]
    assert rel(portions(eng, "p", toks, [1, 1, 2, 1, 3, 1, 1, 1, 1, 2, 5, 1, 20]), want) < TOL["float32"]
    assert rel(portions(eng, "q", toks, [2, 2, 2, 1, 2, 4, 1, 2, 2, 22]), want) < TOL["float32"]
    eng.runner.close()


def test_first_tokens_of_a_sequence():
    """Position 0 sees itself and the sink; the convolutions read zeros in front of it, the scan starts from a zero state."""
    cfg = mixed_model()
    wt = R.random_checkpoint(cfg, 5)
    eng = engine(cfg, wt)
    for n in (1, 2, 3, 4):
        toks = tokens(n, seed=n)
        assert rel(whole(eng, "f", toks), R.forward(cfg, wt, toks)) < TOL["float32"], n
    # the same slot and pages again, now with another first token: nothing of the last request may be read
    toks = tokens(2, seed=9)
    assert rel(whole(eng, "g", toks), R.forward(cfg, wt, toks)) < TOL["float32"]
    eng.runner.close()


@pytest.mark.parametrize("loop", [None, (0, 5, 2), (1, 4, 3), (4, 5, 2), (0, 1, 1), (2, 3, 4)])
def test_residual_stream_after_every_layer_run(loop):
    cfg = dict(mixed_model(), loop=None if loop is None else dict(zip(("start", "stop", "times"), loop)))
    wt = R.random_checkpoint(cfg, 6)
    toks = tokens(30, seed=2)
    eng = engine(cfg, wt)
    eng.runner.layer_probe = []
    got_lg = whole(eng, "p", toks)
    got = eng.runner.layer_probe
    eng.runner.layer_probe = None
    want = []
    want_lg = R.forward(cfg, wt, toks, want)
    assert len(got) == len(want) == len(R.execution_order(cfg))
    for i, (g, x) in enumerate(zip(got, want)):
        assert float((g.double().cpu() - x).abs().max()) < 1e-4 * float(x.abs().max()), i
    assert rel(got_lg, want_lg) < TOL["float32"]
    assert rel(portions(eng, "q", toks, [7, 1, 2, 20]), want_lg) < TOL["float32"]      # without the probe: fused additions
    eng.runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_token_by_token_and_portions_agree(dtype):
    cfg = mixed_model()
    wt = R.random_checkpoint(cfg, 7)
    toks = tokens(90, seed=3)
    want = R.forward(cfg, wt, toks)
    eng = engine(cfg, wt, dtype)
    a = whole(eng, "w", toks)
    b = portions(eng, "t", toks, [1] * 90)
    c = portions(eng, "p", toks, [2, 5, 16, 3, 2, 17, 31, 2, 12])         # page borders (16) inside portions
    for name, got in (("whole", a), ("token by token", b), ("portions", c)):
        assert close(got, want, dtype, cfg), (name, dtype, rel(got, want))
    if dtype == "float32":
        assert rel(b, a) < 1e-5 and rel(c, a) < 1e-5
    eng.runner.close()


def test_long_decoding():
    cfg = mixed_model()
    wt = R.random_checkpoint(cfg, 8)
    toks = tokens(200, seed=4)
    eng = engine(cfg, wt)
    assert rel(portions(eng, "d", toks, [9] + [1] * 191), R.forward(cfg, wt, toks)) < TOL["float32"]
    eng.runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_equal_each_request_alone(dtype):
    cfg = mixed_model()
    wt = R.random_checkpoint(cfg, 9)
    reqs = {"a": tokens(70, seed=1), "b": tokens(33, seed=2), "c": tokens(5, seed=3), "d": tokens(120, seed=4)}
    steps = [[("a", 20), ("b", 30)], [("a", 1), ("b", 1), ("c", 2)], [("a", 2), ("b", 1), ("c", 1), ("d", 50)],
             [("a", 1), ("b", 1), ("c", 1), ("d", 1)], [("a", 46), ("c", 1), ("d", 2)], [("d", 67)]]
    eng = engine(cfg, wt, dtype)
    got = run_steps(eng, reqs, steps)
    for k, toks in reqs.items():
        assert close(got[k], R.forward(cfg, wt, toks), dtype, cfg), (k, dtype)
    assert eng.allocator.num_free == eng.allocator.num_blocks and eng.state_slots.num_free == 4
    eng.runner.close()


def tc_model(all_experts=False):
    """Sizes that take the tensor-core kernels in bf16: GEMM blocks of 64, heads of 64, 128 and 40, chunked scans, expert tiles of
    the grouped GEMM. all_experts: every expert is chosen, so that no rounding flips a choice."""
    top = lambda e, t: e if all_experts else t
    return model_cfg([mamba(heads=4, vdim=64, state=64, groups=2, norm_groups=2, conv=4, mlp=moe(4, top(4, 2), 64)),
                      att(heads=4, kv=2, dim=64, dims=32, scale=0.125, mlp=moe(6, top(6, 1), 128)),
                      att(heads=2, kv=1, dim=128, dims=128, base=15000.0, scale=0.09, conv=3, mlp=moe(2, 2, 64)),
                      mamba(heads=2, vdim=96, state=32, groups=1, norm_groups=1, conv=2),
                      att(heads=8, kv=1, dim=40, dims=16, scale=0.15, conv=2)], width=128, loop=(1, 3, 2))


@pytest.mark.parametrize("all_experts", [True, False])
def test_bf16_portions_on_the_tensor_cores_beside_single_tokens(all_experts):
    """Portions (prompt forms of the attention and scan kernels, the tiled convolutions) beside single tokens (decode forms, several
    key slices, states shifted in place) in one step; portions start and end inside a 64-token chunk and inside pages."""
    cfg = tc_model(all_experts)
    wt = R.random_checkpoint(cfg, 10)
    reqs = {"a": tokens(230, seed=1), "b": tokens(250, seed=2), "c": tokens(240, seed=3)}
    steps = [[("a", 128), ("b", 2)], [("a", 1), ("b", 100), ("c", 70)], [("a", 1), ("b", 1), ("c", 129)], [("a", 1), ("c", 1), ("b", 2)],
             [("a", 99), ("b", 145), ("c", 40)]]
    eng = engine(cfg, wt, "bfloat16", max_model_len=256, max_num_batched_tokens=512, num_gpu_blocks=48, max_logit_rows=512)
    got = run_steps(eng, reqs, steps)
    for k, toks in reqs.items():
        want = R.forward(cfg, wt, toks)
        if all_experts:
            assert close(got[k], want, "bfloat16", cfg), (k, rel(got[k], want))
        else:       # one expert of six, twice in a row through the looped block: a flipped choice replaces a row's feed-forward
            rows = rel_rows(got[k], want)
            assert float(rows.quantile(0.8)) < TOL["bfloat16"] and float(rows.max()) < 1.5, (k, rows.quantile(0.8), rows.max())
    eng.runner.close()


def test_a_step_of_hundreds_of_rows_mixes_single_tokens_and_portions_in_fp32():
    """More than 256 rows in a step: the tiled forms of both convolutions, with decoded tokens whose states shift in place."""
    cfg = mixed_model()
    wt = R.random_checkpoint(cfg, 16)
    reqs = {"a": tokens(40, seed=1), "b": tokens(310, seed=2), "c": tokens(20, seed=3)}
    steps = [[("a", 11), ("b", 3), ("c", 2)], [("a", 1), ("c", 1), ("b", 300)], [("b", 1), ("a", 1), ("c", 2)], [("a", 27), ("b", 6), ("c", 15)]]
    eng = engine(cfg, wt, max_model_len=320, max_num_batched_tokens=512, max_logit_rows=512)
    got = run_steps(eng, reqs, steps)
    for k, toks in reqs.items():
        assert rel(got[k], R.forward(cfg, wt, toks)) < TOL["float32"], k
    eng.runner.close()


def test_pages_and_slots_are_reused_without_leaking_old_state():
    cfg = mixed_model()
    wt = R.random_checkpoint(cfg, 12)
    eng = engine(cfg, wt, num_gpu_blocks=10, max_num_seqs=2, max_model_len=128)
    for rnd in range(4):
        a, b = tokens(60 + rnd, seed=20 + rnd), tokens(17 + 3 * rnd, seed=30 + rnd)
        got = run_steps(eng, {"a": a, "b": b}, [[("a", 30), ("b", len(b) - 2)], [("a", 1), ("b", 2)], [("a", len(a) - 31)]])
        assert rel(got["a"], R.forward(cfg, wt, a)) < TOL["float32"], rnd
        assert rel(got["b"], R.forward(cfg, wt, b)) < TOL["float32"], rnd
    assert eng.allocator.num_free == eng.allocator.num_blocks and eng.state_slots.num_free == 2
    eng.runner.close()


ODD = {
    "no_loop_no_cap_unit_scale": lambda: model_cfg([att(mlp=moe()), mamba()], mult=1.0, cap=None),
    "no_experts_anywhere": lambda: model_cfg([att(), mamba(), att(heads=1, kv=1)], loop=(0, 3, 2)),
    "only_recurrent_layers": lambda: model_cfg([mamba(), mamba(heads=1, vdim=5, state=3, groups=1, mlp=moe())], loop=(1, 2, 3)),
    "only_attention": lambda: model_cfg([att(mlp=moe(2, 1, 8)), att(heads=5, kv=5, dim=6, dims=6, conv=1)]),
    "tight_cap": lambda: model_cfg([att(mlp=moe())], cap=0.75),
    "widths_off_every_block": lambda: model_cfg([mamba(heads=3, vdim=7, state=5, groups=3, norm_groups=3, mlp=moe(3, 2, 7)),
                                                 att(heads=3, kv=1, dim=5, dims=2, mlp=moe(2, 1, 9))], width=54, vocab=77, loop=(0, 2, 2)),
    "width_without_vectors": lambda: model_cfg([att(mlp=moe()), mamba(mlp=moe(3, 1, 5))], width=51, vocab=61, loop=(1, 2, 2)),
    "large_eps": lambda: model_cfg([mamba(mlp=moe()), att()], eps=0.3),
    "many_experts": lambda: model_cfg([mamba(mlp=moe(70, 9, 8))]),
    "wide_ff_narrow_model": lambda: model_cfg([att(mlp=moe(2, 2, 300))], width=32),
    "long_rotation_base": lambda: model_cfg([att(dim=16, dims=16, base=1000000.0), att(dim=16, dims=2, base=1.5)]),
}


@pytest.mark.parametrize("name", sorted(ODD))
def test_odd_configurations_whole_and_in_portions(name):
    cfg = ODD[name]()
    wt = R.random_checkpoint(cfg, 14)
    toks = tokens(75, vocab=cfg["vocab"], seed=5)
    want = R.forward(cfg, wt, toks)
    for dtype in ("float32", "bfloat16"):
        eng = engine(cfg, wt, dtype)
        assert close(whole(eng, "w", toks), want, dtype, cfg), (name, dtype)
        assert close(portions(eng, "p", toks, [3, 2, 30, 1, 1, 38]), want, dtype, cfg), (name, dtype)
        eng.runner.close()


def drawn_model(seed):
    g = torch.Generator().manual_seed(seed)

    def ri(lo, hi):
        return int(torch.randint(lo, hi + 1, (1,), generator=g))

    layers = []
    for i in range(ri(1, 5)):
        E = ri(1, 9)
        mlp = moe(E, ri(1, min(4, E)), [64, ri(4, 80)][ri(0, 1)]) if ri(0, 2) else None
        if ri(0, 1):
            kv = ri(1, 4)
            dim = [8 * ri(1, 16), ri(2, 40)][ri(0, 1)]
            layers.append(att(heads=kv * ri(1, 3), kv=kv, dim=dim, dims=2 * ri(0, dim // 2), base=float(ri(10, 100000)),
                              scale=0.02 * ri(1, 20), conv=ri(1, 6), mlp=mlp))
        else:
            G, h = ri(1, 3), ri(1, 2)
            R_ = ri(1, 2)
            layers.append(mamba(heads=G * h, vdim=R_ * ri(1, 36), state=[32, 64, ri(1, 80)][ri(0, 2)], groups=G, norm_groups=R_,
                                conv=ri(1, 6), mlp=mlp))
    a = ri(0, len(layers) - 1)
    loop = (a, ri(a + 1, len(layers)), ri(1, 3)) if ri(0, 2) else None
    return model_cfg(layers, width=[64 * ri(1, 3), ri(24, 120)][ri(0, 1)], vocab=ri(30, 200), loop=loop, mult=0.1 * ri(3, 12),
                     cap=float(ri(2, 40)))


@pytest.mark.parametrize("draw", range(10))
def test_drawn_models_whole_cut_and_mixed(draw):
    cfg = drawn_model(300 + draw)
    wt = R.random_checkpoint(cfg, 400 + draw)
    V = cfg["vocab"]
    reqs = {"a": tokens(80, V, seed=1), "b": tokens(47, V, seed=2), "c": tokens(9, V, seed=3)}
    want = torch.cat([R.forward(cfg, wt, v) for v in reqs.values()])
    steps = [[("a", 17), ("c", 2)], [("a", 1), ("b", 31), ("c", 1)], [("a", 2), ("b", 1), ("c", 1)], [("a", 60), ("b", 15), ("c", 5)]]
    for dtype in ("float32", "bfloat16"):
        eng = engine(cfg, wt, dtype)
        alone = np.concatenate([eng.feed([(k, v, list(range(len(v))))], [k]) for k, v in reqs.items()])
        got = run_steps(eng, reqs, steps)
        got = np.concatenate([got[k] for k in reqs])
        for x in (alone, got):
            rows = rel_rows(x, want)
            if dtype == "float32":       # tiny heads amplify rounding through their norm on single rows
                assert float(rows.quantile(0.9)) < TOL[dtype] and float(rows.max()) < 4e-4, (draw, cfg, float(rows.max()))
            else:
                assert float(rows.quantile(0.6 if chooses(cfg) else 0.95)) < TOL[dtype] and float(rows.max()) < 1.2, (draw, cfg, rows.quantile(0.6), rows.max())
        if dtype == "float32":      # the cut must not matter, whatever the conditioning
            assert rel(got, alone) < 2e-4, (draw, cfg)
        eng.runner.close()


# ---- models built so that a fault shows ---------------------------------------------------------------------------------------

def pointed_model(dim=32, pos_free=True):
    """One attention layer (no experts) in which the query of token 0 scores the key of token 1 far above every other key: W_q maps
    token 0's normed embedding onto W_k's image of token 1's. Taps pass the row itself, so the value is that key."""
    cfg = model_cfg([att(heads=2, kv=1, dim=dim, dims=0 if pos_free else dim // 2, base=10.0, scale=24.0 / dim, conv=2)], width=64)
    wt = R.random_checkpoint(cfg, 19)
    eps = 1e-5
    u = R.centred_norm(wt["embed"], wt["l0.norm1"], eps)
    a, b = u[0], u[1]
    k_b = wt["l0.mix.k"] @ b
    for h in range(2):
        q = wt["l0.mix.q"][h * dim:(h + 1) * dim]
        q += torch.outer(4.0 * k_b - q @ a, a) / (a @ a)
    for n in ("q", "k"):
        t = torch.zeros_like(wt[f"l0.mix.{n}.conv"])
        t[:, -1] = 1.0
        wt[f"l0.mix.{n}.conv"] = t
    wt["l0.mix.o"] = wt["l0.mix.o"] * 3.0
    return cfg, {k: t.to(torch.bfloat16).to(F64) for k, t in wt.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_among_hundreds_is_found_at_every_place(dtype):
    """The pointed-at key sits at the first token, on both sides of page borders, at the edges of a prompt portion and in the last
    row in front of the query; the query comes in a prompt and as a decoded token, with several key slices in flight."""
    cfg, wt = pointed_model()
    eng = engine(cfg, wt, dtype, max_model_len=512, max_num_batched_tokens=512, num_gpu_blocks=64, max_logit_rows=16)
    n = 400
    base = [t + 2 if t < 2 else t for t in tokens(n, seed=12)]
    plain = R.forward(cfg, wt, base + [0])[-1]
    for place in (0, 1, 15, 16, 17, 127, 128, 255, 256, 383, 398, 399):
        toks = list(base)
        toks[place] = 1
        toks.append(0)
        want = R.forward(cfg, wt, toks)[-1]
        assert float(rel_rows(want[None], plain[None])) > 0.2          # the reference itself: the key at `place` decides the row
        rows = [eng.feed([("w", toks, [n])], ["w"])]
        eng.feed([("d", toks[:n], [])])
        rows.append(eng.feed([("d", toks[n:], [0])], ["d"]))
        eng.feed([("c", toks[:128], [])])
        eng.feed([("c", toks[128:256], [])])
        rows.append(eng.feed([("c", toks[256:], [n - 256])], ["c"]))
        eng.feed([("e", toks[:n - 1], [])])
        rows.append(eng.feed([("e", toks[n - 1:], [1])], ["e"]))
        for i, got in enumerate(rows):
            assert rel(got, want[None]) < (1e-4 if dtype == "float32" else 0.06), (place, i, rel(got, want[None]))
    eng.runner.close()


def test_rotated_far_keys_depend_on_their_distance():
    cfg, wt = pointed_model(pos_free=False)
    eng = engine(cfg, wt, max_logit_rows=16)
    rows = []
    for place in (3, 4, 60, 119):
        toks = [t + 2 if t < 2 else t for t in tokens(120, seed=13)] + [0]
        toks[place] = 1
        want = R.forward(cfg, wt, toks)[-1:]
        got = eng.feed([("r", toks[:77], [])])
        got = eng.feed([("r", toks[77:], [43])], ["r"])
        assert rel(got, want) < 1e-4, place
        rows.append(want)
    assert rel(rows[2], rows[3]) > 0.02
    eng.runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_sink_takes_its_share_whatever_the_scores(dtype):
    """Small scores and few keys: the sink holds 1 / (1 + n) of the weight. Without it the mixer's output would be 1 + 1/n times as
    large, which the reference shows to move the logits by far more than the tolerance."""
    cfg = model_cfg([att(heads=2, kv=2, dim=64, dims=32, scale=0.003)], width=64)
    wt = R.random_checkpoint(cfg, 24)
    wt["l0.mix.o"] = wt["l0.mix.o"] * 4.0
    toks = tokens(6, seed=5)
    want = R.forward(cfg, wt, toks)
    eng = engine(cfg, wt, dtype)
    tol = TOL["float32"] if dtype == "float32" else 0.03
    assert rel(whole(eng, "w", toks), want) < tol
    assert rel(portions(eng, "d", toks, [1] * 6), want) < tol
    no_sink = dict(wt, **{"l0.mix.o": wt["l0.mix.o"] * 2.0})
    assert rel(R.forward(cfg, no_sink, toks[:1]), want[:1]) > 0.1      # position 0: half the weight is the sink's
    eng.runner.close()


def test_a_state_that_barely_decays_carries_far_tokens_across_steps_and_slots():
    cfg = model_cfg([mamba(heads=2, vdim=8, state=8, groups=1), mamba(heads=2, vdim=16, state=32, groups=2, mlp=moe(2, 2, 16))], loop=(0, 2, 2))
    wt = R.random_checkpoint(cfg, 22)
    for i in range(2):
        wt[f"l{i}.mix.A_log"] = torch.full_like(wt[f"l{i}.mix.A_log"], -9.0)
        wt[f"l{i}.mix.dt_bias"] = torch.full_like(wt[f"l{i}.mix.dt_bias"], -1.0)
    a, b = tokens(230, seed=7), tokens(190, seed=8)
    wa, wb = R.forward(cfg, wt, a), R.forward(cfg, wt, b)
    short = R.forward(cfg, wt, a[100:])             # the reference itself: the last rows depend on the first hundred tokens
    assert rel(short[-10:], wa[-10:]) > 0.05
    eng = engine(cfg, wt, max_num_seqs=2)
    got = run_steps(eng, {"a": a, "b": b}, [[("a", 64), ("b", 3)], [("a", 65), ("b", 1)], [("a", 1), ("b", 128)],
                                            [("a", 1), ("b", 1)], [("a", 99), ("b", 57)]])
    assert rel(got["a"], wa) < TOL["float32"] and rel(got["b"], wb) < TOL["float32"]
    # the slots again, from position 0: the old states must be gone
    got = run_steps(eng, {"c": b[:40], "d": a[:50]}, [[("c", 40), ("d", 2)], [("d", 48)]])
    assert rel(got["c"], wb[:40]) < TOL["float32"] and rel(got["d"], wa[:50]) < TOL["float32"]
    eng.runner.close()


def test_bf16_chunked_scan_matches_decoding_with_strong_and_weak_decays():
    for a_log, dt_b in ((-6.0, 0.0), (0.0, -2.0), (3.0, 2.0)):
        cfg = model_cfg([mamba(heads=2, vdim=64, state=64, groups=1, conv=4)], width=128)
        wt = R.random_checkpoint(cfg, 23)
        wt["l0.mix.A_log"] = torch.full_like(wt["l0.mix.A_log"], a_log)
        wt["l0.mix.dt_bias"] = torch.full_like(wt["l0.mix.dt_bias"], dt_b)
        toks = tokens(200, seed=9)
        want = R.forward(cfg, wt, toks)
        eng = engine(cfg, wt, "bfloat16")
        got = portions(eng, "p", toks, [70, 1, 1, 100, 2, 26])
        assert close(got, want, "bfloat16", cfg), (a_log, dt_b, rel(got, want))
        eng.runner.close()


# ---- generation through the framework's own entry point -----------------------------------------------------------------------

@pytest.mark.parametrize("mode", ["plain", "chunked_prefill", "async", "graphs"])
def test_greedy_generation_matches_the_reference(mode):
    from atx.scheduler import SamplingParams

    cfg = mixed_model()
    wt = R.random_checkpoint(cfg, 13)
    prompts = [tokens(37, seed=1), tokens(5, seed=2), tokens(64, seed=3)]
    kw = {"plain": {}, "chunked_prefill": {"max_num_batched_tokens": 16}, "async": {"async_scheduling": True},
          "graphs": {"async_scheduling": True, "enable_cuda_graphs": True}}[mode]
    eng = engine(cfg, wt, **kw)
    outs = eng.generate_sync(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        lg = R.forward(cfg, wt, p + o[:-1])[len(p) - 1:]
        top2 = lg.topk(2, dim=-1).values
        for i, tok in enumerate(o):            # teacher-forced: every token is the reference's arg-max (ties aside)
            assert tok == int(lg[i].argmax()) or float(top2[i, 0] - top2[i, 1]) < 1e-4, (mode, i)
    assert eng.allocator.num_free == eng.allocator.num_blocks and eng.state_slots.num_free == 4
    eng.runner.close()


@pytest.mark.parametrize("mode", ["plain", "graphs"])
def test_bf16_greedy_generation_on_the_tensor_core_kernels(mode):
    """Graph replay runs the experts on a second branch beside the mixer."""
    from atx.scheduler import SamplingParams

    cfg = tc_model(all_experts=True)      # a choice between experts that bf16 rounding flips would move whole rows
    wt = R.random_checkpoint(cfg, 17)
    prompts = [tokens(100, seed=1), tokens(5, seed=2), tokens(64, seed=3)]
    kw = {"plain": {}, "graphs": {"async_scheduling": True, "enable_cuda_graphs": True}}[mode]
    eng = engine(cfg, wt, "bfloat16", **kw)
    outs = eng.generate_sync(prompts, SamplingParams(temperature=0.0, max_tokens=60, ignore_eos=True))
    near = 0
    for p, o in zip(prompts, outs):
        assert len(o) == 60
        lg = R.forward(cfg, wt, p + o[:-1])[len(p) - 1:]
        spread = float(lg.std())
        top2 = lg.topk(2, dim=-1).values
        for i, tok in enumerate(o):
            if tok != int(lg[i].argmax()):
                near += 1
                assert float(top2[i, 0] - lg[i, tok]) < 0.15 * spread, (mode, i)
    assert near <= 12
    assert eng.allocator.num_free == eng.allocator.num_blocks
    eng.runner.close()


def test_named_shape_generates_through_the_registry():
    from atx.config import EngineConfig, resolve_model
    from atx.engine import LLMEngine
    from atx.scheduler import SamplingParams

    src = resolve_model("random:lifuzen-tiny:3")
    ecfg = EngineConfig(max_model_len=128, max_num_seqs=4, max_num_batched_tokens=128, num_gpu_blocks=32,
                        enable_prefix_caching=False, enable_cuda_graphs=True, async_scheduling=True)
    eng = LLMEngine(src, ecfg)
    outs = eng.generate_sync([tokens(40, 1024, 1), tokens(3, 1024, 2)], SamplingParams(temperature=0.0, max_tokens=8,
                                                                                      ignore_eos=True))
    assert [len(o) for o in outs] == [8, 8] and all(0 <= t < 1024 for o in outs for t in o)
    eng.runner.close()


# ---- kernels alone ------------------------------------------------------------------------------------------------------------

def lib():
    from atx import _cabi

    return _cabi.load(), _cabi


def ck(rc):
    L, _ = lib()
    assert rc == 0, L.atx_last_error().decode()


def dev(t, dtype=None):
    return torch.as_tensor(t).to(device=DEV, dtype=dtype).contiguous() if dtype else torch.as_tensor(t).to(DEV).contiguous()


def stream():
    return torch.cuda.current_stream().cuda_stream


def types(dtype):
    _, Cb = lib()
    return (torch.float32, Cb.DT_F32) if dtype == "float32" else (torch.bfloat16, Cb.DT_BF16)


def seq_view(counts, pos0, slots):
    """Device arrays of a step whose sequences hold `counts` consecutive rows each."""
    starts = np.concatenate([[0], np.cumsum(counts)[:-1]]).astype(np.int32)
    tok_seq = np.concatenate([np.full(c, i, np.int32) for i, c in enumerate(counts)])
    i32 = torch.int32
    return (dev(tok_seq, i32), dev(starts, i32), dev(np.asarray(counts, np.int32), i32), dev(np.asarray(pos0, np.int32), i32),
            dev(np.asarray(slots, np.int32), i32))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,T", [(40, 5), (38, 7), (1024, 3), (2048, 600), (4096, 530), (8192, 520), (12288, 2), (12288, 515)])
def test_parallel_residual_with_experts_an_entering_row_and_two_norms(W, T, dtype):
    L, Cb = lib()
    xt, dt = types(dtype)
    tol = 2e-5 if dtype == "float32" else 0.01
    g = torch.Generator().manual_seed(W + T)
    V, top, P = 11, 3, 3 * T
    h0, y0, ye = (torch.randn(n, W, generator=g).float() for n in (T, T, P))
    table = torch.randn(V, W, generator=g).to(xt)
    vec, wa, wb = ((0.2 * torch.randn(W, generator=g)).to(xt) for _ in range(3))
    ids = torch.randint(0, V, (T,), generator=g, dtype=torch.int32)
    wgt = torch.rand(T, top, generator=g).float()
    slot_of = torch.randperm(P, generator=g).to(torch.int32).view(T, top).clone()
    slot_of[0, 1] = -1
    w = torch.where(slot_of >= 0, wgt, torch.zeros(())).double()
    mix = (w[:, :, None] * ye.double()[slot_of.clamp(min=0).long()]).sum(1)
    eps = 1e-3
    tabd, vecd, wad, wbd, idd, yed, wgd, sld = (dev(t) for t in (table, vec, wa, wb, ids, ye, wgt, slot_of))

    def norm(v, wt):
        return R.centred_norm(v, wt.double(), eps)

    def run(h, y=None, experts=False, mode=0, vec=False, a=True, b=True, rows=None, zero_y=0, zero=None):
        t = Cb.ResidTerms()
        t.y_scale, t.table_mode, t.vocab, t.zero_y = 0.7, mode, V, zero_y
        t.ids, t.table, t.vec = idd.data_ptr(), tabd.data_ptr(), vecd.data_ptr() if vec else None
        t.y = None if y is None else y.data_ptr()
        if experts:
            t.experts, t.wgt, t.slot_of, t.lde, t.top = yed.data_ptr(), wgd.data_ptr(), sld.data_ptr(), W, top
        n = T if rows is None else len(rows)
        oa, ob = torch.zeros(n, W, dtype=xt, device=DEV), torch.zeros(n, W, dtype=xt, device=DEV)
        rd = None if rows is None else dev(torch.tensor(rows, dtype=torch.int32))
        ck(L.atx_parallel_resid_norm(h.data_ptr(), ctypes.byref(t), wad.data_ptr() if a else None, oa.data_ptr() if a else None,
                                     wbd.data_ptr() if b else None, ob.data_ptr() if b else None, 1.0, None if rd is None else rd.data_ptr(),
                                     n, W, eps, None if zero is None else zero.data_ptr(), 0 if zero is None else zero.numel() * 4, dt, 0, stream()))
        torch.cuda.synchronize()
        return oa.double().cpu(), ob.double().cpu()

    def near(got, want, t=tol):
        assert float((got - want).abs().max()) < t * max(1.0, float(want.abs().max())), float((got - want).abs().max())

    hd = torch.full((T, W), 9.0, device=DEV)
    oa, ob = run(hd, mode=2, vec=True)                                                      # the stream starts as the embedding row
    v = table.double()[ids.long()] + vec.double()
    near(hd.double().cpu(), v, 2e-6), near(oa, norm(v, wa)), near(ob, norm(v, wb))
    hd, yd, zero = dev(h0), dev(y0), torch.full((4 * 300,), 5.0, device=DEV)
    oa, ob = run(hd, y=yd, experts=True, mode=1, vec=True, zero_y=1, zero=zero)               # everything at once
    v = h0.double() + 0.7 * (y0.double() + mix) + table.double()[ids.long()] + vec.double()
    near(hd.double().cpu(), v, 2e-6), near(oa, norm(v, wa)), near(ob, norm(v, wb))
    assert float(yd.abs().max()) == 0.0 and float(zero.abs().max()) == 0.0
    hd, yd = dev(h0), dev(y0)
    oa, ob = run(hd, y=yd, b=False)                                                         # a layer without experts, one norm
    v = h0.double() + 0.7 * y0.double()
    near(hd.double().cpu(), v, 2e-6), near(oa, norm(v, wa))
    assert float(ob.abs().max()) == 0.0 and torch.equal(yd.cpu(), y0)
    rows = [T - 1, 0, T - 1]
    hd = dev(h0)
    oa, _ = run(hd, y=yd, experts=True, b=False, rows=rows)                                  # gathered rows: the stream is only read
    near(oa, norm(h0.double() + 0.7 * (y0.double() + mix), wa)[rows])
    assert torch.equal(hd.cpu(), h0)
    run(hd, y=yd, experts=True, a=False, b=False)                                            # no norm: only the addition
    near(hd.double().cpu(), h0.double() + 0.7 * (y0.double() + mix), 2e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("K,H,G,D,rd,T", [(4, 3, 2, 64, 32, 60), (4, 2, 1, 128, 128, 700), (3, 4, 4, 32, 8, 300), (2, 2, 1, 256, 64, 270),
                                          (7, 2, 2, 96, 0, 40), (1, 2, 1, 16, 16, 300), (4, 2, 1, 7, 4, 30), (11, 1, 1, 64, 2, 40), (3, 1, 1, 300, 300, 20)])
def test_convolved_heads_across_steps_slots_and_pages(K, H, G, D, rd, T, dtype):
    """Two sequences through steps of several sizes (single rows shift their state in place, longer ones through the update
    kernel), padded rows at the end, junk in slots and pages: queries, normed rotated keys and raw keys of every position."""
    L, Cb = lib()
    from atx.models.common import rotation_table

    xt, dt = types(dtype)
    tol = 2e-5 if dtype == "float32" else 0.01
    g = torch.Generator().manual_seed(K * 1000 + D)
    C, bs, eps = (H + G) * D, 16, 1e-4
    n = {"a": T, "b": T // 2 + 3}
    x = {k: torch.randn(m, C, generator=g).float() for k, m in n.items()}
    w = torch.randn(C, K, generator=g).to(xt)
    want = {}
    for k, v in x.items():
        u = R.causal_taps(v.double(), w.double())
        q, kk = u[:, :H * D].reshape(-1, H, D), u[:, H * D:].reshape(-1, G, D)
        rot = (lambda t: R.rotate_pairs(t, rd, 40.0)) if rd else (lambda t: t)
        want[k] = (R.unit_rms(rot(q), eps), R.unit_rms(rot(kk), eps), kk)
    table = rotation_table(40.0, rd, max(n.values()) + 1, torch.device(DEV)) if rd else None
    nblk = {k: (m + bs - 1) // bs for k, m in n.items()}
    perm = torch.randperm(sum(nblk.values()) + 2, generator=g).tolist()
    blocks = {"a": perm[:nblk["a"]], "b": perm[nblk["a"]:nblk["a"] + nblk["b"]]}
    kc, vc = (torch.full((len(perm), G, bs, D), 7.0, dtype=xt, device=DEV) for _ in range(2))
    state = torch.full((3, max(1, K - 1), C), 77.0, device=DEV)
    wd, slot = dev(w), {"a": 2, "b": 0}
    at, got_q = {"a": 0, "b": 0}, {"a": [], "b": []}
    for step in [{"b": 3, "a": 1}, {"a": 1, "b": 1}, {"a": 2}, {"b": 1, "a": T // 3}, {"a": 1, "b": 2}, {"b": 1, "a": T}, {"b": T}]:
        live = [(k, min(c, n[k] - at[k])) for k, c in step.items() if at[k] < n[k]]
        live.sort(key=lambda kc_: kc_[1] != 1)                        # single rows in front, as a step is laid out
        if not live:
            continue
        inplace = sum(1 for _, c in live if c == 1)
        rows = torch.cat([x[k][at[k]:at[k] + c] for k, c in live] + [torch.full((2, C), 3.0)])
        pos = np.concatenate([np.arange(at[k], at[k] + c) for k, c in live] + [[0, 0]]).astype(np.int32)
        slots = np.concatenate([[blocks[k][p // bs] * bs + p % bs for p in range(at[k], at[k] + c)] for k, c in live] + [[-1, -1]]).astype(np.int32)
        tok_seq, starts, cnt, pos0, sl = seq_view([c for _, c in live], [at[k] for k, _ in live], [slot[k] for k, _ in live])
        tok_seq = torch.cat([tok_seq, torch.full((2,), -1, dtype=torch.int32, device=DEV)])
        q = torch.zeros(len(rows), H * D, dtype=xt, device=DEV)
        src = torch.zeros(len(rows), C + 8, device=DEV)               # the slices start at column 4 of a wider row
        src[:, 4:4 + C] = rows.to(DEV)
        tp = None if table is None else table.data_ptr()
        esz = 4 if dtype == "float32" else 2
        segs = Cb.conv_head_segs(Cb.ConvHeadSeg(src_off=4, heads=H, width=D, norm=1, rot_dims=rd, dst_kind=Cb.HEAD_DST_ROWS, w=wd.data_ptr(), rot=tp,
                                                dst=q.data_ptr(), dst_ld=H * D),
                                 Cb.ConvHeadSeg(src_off=4 + H * D, heads=G, width=D, norm=1, rot_dims=rd, dst_kind=Cb.HEAD_DST_PAGES,
                                                w=wd.data_ptr() + H * D * K * esz, rot=tp, dst=kc.data_ptr(), raw_dst=vc.data_ptr()))
        posd, slotd = dev(pos), dev(slots)
        ck(L.atx_conv_head_prepare(src.data_ptr(), C + 8, segs, 2, K, state.data_ptr(), C, inplace, posd.data_ptr(), slotd.data_ptr(),
                                   tok_seq.data_ptr(), starts.data_ptr(), pos0.data_ptr(), sl.data_ptr(), len(rows), bs, eps, dt, 0, stream()))
        if len(live) > inplace:
            o = 4 * inplace
            ck(L.atx_conv_state_update(src.data_ptr(), C + 8, 4, state.data_ptr(), starts.data_ptr() + o, cnt.data_ptr() + o, pos0.data_ptr() + o,
                                       sl.data_ptr() + o, len(live) - inplace, C, K, 0, stream()))
        torch.cuda.synchronize()
        o = 0
        for k, c in live:
            got_q[k].append(q[o:o + c].double().cpu())
            o += c
            at[k] += c
        assert float(q[o:].float().abs().max()) == 0.0                # padded rows are left alone
    assert at == n
    for k in n:
        wq, wk, wv = want[k]
        assert float((torch.cat(got_q[k]).view(-1, H, D) - wq).abs().max()) < tol * float(wq.abs().max()), k
        idx = [(blocks[k][p // bs], p % bs) for p in range(n[k])]
        gk = torch.stack([kc[b_, :, o_] for b_, o_ in idx]).double().cpu()
        gv = torch.stack([vc[b_, :, o_] for b_, o_ in idx]).double().cpu()
        assert float((gk - wk).abs().max()) < tol * float(wk.abs().max()) and float((gv - wv).abs().max()) < tol * float(wv.abs().max()), k
    assert float((kc[perm[-1]] - 7.0).abs().max()) == 0.0 and float((vc[perm[-2]] - 7.0).abs().max()) == 0.0


@pytest.mark.parametrize("K,C,H,T", [(4, 40, 3, 20), (4, 300, 5, 400), (2, 7, 1, 9), (8, 64, 4, 300), (1, 16, 2, 20), (11, 24, 2, 30)])
def test_scan_convolution_shifts_single_row_states_in_place(K, C, H, T):
    """The in-place form against the two-launch form on the same steps: outputs and states, bit for bit."""
    L, Cb = lib()
    g = torch.Generator().manual_seed(K + C)
    w, b, db, al = (torch.randn(*s, generator=g).float().to(DEV) for s in ((C, K), (C,), (H,), (H,)))
    states = [torch.full((4, max(1, K - 1), C), 5.0, device=DEV) for _ in range(2)]
    pos = {0: 0, 1: 0, 2: 0}
    for counts in ([1, 3, 1], [1, 1, 1], [1, T, 2], [1, 1, T]):
        order = sorted(range(3), key=lambda i: counts[i] != 1)
        cs = [counts[i] for i in order]
        tok_seq, starts, cnt, pos0, sl = seq_view(cs, [pos[i] for i in order], [3 - i for i in order])
        n_in = sum(1 for c in cs if c == 1)
        src = torch.randn(sum(cs), C + H + 2, generator=g).float().to(DEV)
        outs = []
        for st, inplace in zip(states, (0, n_in)):
            o = [torch.zeros(sum(cs), m, device=DEV) for m in (C, H, H)]
            ck(L.atx_conv_dt_inplace(src.data_ptr(), C + H + 2, 1, C + 1, w.data_ptr(), b.data_ptr(), db.data_ptr(), al.data_ptr(), st.data_ptr(),
                                     *(t.data_ptr() for t in o), tok_seq.data_ptr(), starts.data_ptr(), pos0.data_ptr(), sl.data_ptr(), inplace,
                                     sum(cs), C, H, K, Cb.DT_F32, 0, stream()))
            f = 4 * inplace
            if len(cs) > inplace:
                ck(L.atx_conv_state_update(src.data_ptr(), C + H + 2, 1, st.data_ptr(), starts.data_ptr() + f, cnt.data_ptr() + f,
                                           pos0.data_ptr() + f, sl.data_ptr() + f, len(cs) - inplace, C, K, 0, stream()))
            torch.cuda.synchronize()
            outs.append(o)
        assert all(torch.equal(p, q) for p, q in zip(*outs)) and torch.equal(*states)
        for i in range(3):
            pos[i] += counts[i]


def test_sigmoid_routing_keeps_scores_and_orders_saturated_ones_by_their_logits():
    L, Cb = lib()
    g = torch.Generator().manual_seed(2)
    z = (torch.randn(33, 40, generator=g) * 4).float()
    z[0, :37] = 30.0 + torch.arange(37).float()           # every sigmoid is 1 in fp32: the logits still order them
    for top, normalize, power, scale in ((1, 0, 2, 1.0), (5, 0, 2, 1.0), (37, 0, 1, 1.5), (4, 1, 1, 1.75), (4, 1, 2, 0.5)):
        sel, wgt, zd = torch.zeros(33, top, dtype=torch.int32, device=DEV), torch.zeros(33, top, device=DEV), dev(z)
        ck(L.atx_moe_route_scored(zd.data_ptr(), 40, None, 37, top, scale, normalize, Cb.MOE_SIGMOID, power, sel.data_ptr(), wgt.data_ptr(), 33, 0, stream()))
        torch.cuda.synchronize()
        idx = z[:, :37].topk(top, -1).indices
        assert torch.equal(sel.cpu().long(), idx)
        val = torch.sigmoid(z[:, :37].double()).gather(1, idx)
        if normalize:
            val = val / val.sum(-1, keepdim=True)
        assert float((wgt.double().cpu() - (val * scale) ** power).abs().max()) < 1e-5, (top, normalize, power)


@pytest.mark.parametrize("T", [1, 3, 16, 17, 50, 64, 90, 700])
def test_squared_relu_experts_decode_tiles_and_the_grouped_gemm(T):
    """The helper the program uses, both dtypes, both tile sizes and the tcgen05 path: by-slot outputs, summed with squared scores,
    against the definition (the weight on the expert's input)."""
    from atx.models.common import Experts

    L, Cb = lib()
    for E, top, F, W in ((5, 2, 64, 128), (3, 3, 192, 64), (9, 1, 40, 72), (160, 2, 320, 64), (2, 1, 512, 1024)):
        g = torch.Generator().manual_seed(T + E)
        wt = {f"e{e}.{n}": (torch.randn(*s, generator=g, dtype=F64) * s[1] ** -0.5).to(torch.bfloat16).to(F64)
              for e in range(E) for n, s in (("up", (F, W)), ("down", (W, F)))}
        wt["router"] = torch.randn(E, W, generator=g, dtype=F64) * 0.3
        x = torch.randn(T, W, generator=g, dtype=F64).to(torch.bfloat16).to(F64)
        want = R.expert_mixture(x, {"router": {"top": top}}, wt, "")
        logits = dev((x @ wt["router"].T).float())
        for dtype in ("float32", "bfloat16"):
            xt, dt = types(dtype)
            xn = torch.zeros(max(T, 16), W, dtype=xt, device=DEV)
            xn[:T] = x.to(xt)
            ex = Experts(L, ck, [{"router": {"top": top, "experts": E}, "expert": {"ff": F}}], max(T, 16), W, xn, dt, power=2)
            up = torch.stack([wt[f"e{e}.up"] for e in range(E)]).to(device=DEV, dtype=xt).contiguous()
            down = torch.stack([wt[f"e{e}.down"] for e in range(E)]).to(device=DEV, dtype=xt).contiguous()
            n = ex.run(logits.data_ptr(), E, top, up, down, ex.plans(up, down), T, T <= 64, 0, stream())
            torch.cuda.synchronize()
            assert n == (3 if T <= 64 else 5 if dtype == "bfloat16" and W % 64 == 0 and F % 64 == 0 else 4)
            out = ex.out.view(-1, W).double().cpu()
            sl, wg = ex.slot_of[:T * top].long().cpu().view(T, top), ex.wgt[:T * top].double().cpu().view(T, top)
            assert sorted(sl.flatten().tolist()) == list(range(T * top))
            got = (wg[:, :, None] * out[sl]).sum(1)
            assert float((got - want).abs().max()) < (1e-4 if dtype == "float32" else 0.03) * float(want.abs().max()), (E, dtype)


@pytest.mark.parametrize("T,N,K", [(3, 1000, 128), (40, 300, 512), (100, 257, 64), (300, 520, 128)])
def test_gemm_with_a_capped_store(T, N, K):
    L, Cb = lib()
    g = torch.Generator().manual_seed(T)
    w = (3.0 * torch.randn(N, K, generator=g)).to(torch.bfloat16)
    x = torch.zeros(max(T, 16), K, dtype=torch.bfloat16, device=DEV)
    x[:T] = torch.randn(T, K, generator=g).to(torch.bfloat16).to(DEV)
    plan = Cb.GemmPlan(dev(w), x)
    plan.set_gate(1.0, 20.0, 0.0)
    out = torch.full((T, N + 4), 3.0, device=DEV)
    plan.run(out, T, Cb.GEMM_SOFTCAP_F32, splits=1)
    torch.cuda.synchronize()
    z = x[:T].cpu().double() @ w.double().T
    assert float((z.abs() > 20.0).double().mean()) > 0.3                # the cap bites
    assert float((out[:, :N].double().cpu() - 20.0 * torch.tanh(z / 20.0)).abs().max()) < 1e-3
    assert float((out[:, N:] - 3.0).abs().max()) == 0.0
    y = dev(z.float())
    ck(L.atx_soft_cap(y.data_ptr(), N, T, N - 3, 20.0, 0, stream()))     # the kernel of the fp32 path, a few columns left out
    torch.cuda.synchronize()
    assert float((y[:, :N - 3].double().cpu() - 20.0 * torch.tanh(z[:, :N - 3] / 20.0)).abs().max()) < 1e-4
    assert torch.equal(y[:, N - 3:].cpu(), z[:, N - 3:].float())


# ---- the replay command -------------------------------------------------------------------------------------------------------

def write_checkpoint(folder, cfg, wt):
    """config.json + model.safetensors (bf16): an 8-byte length, a JSON header of name -> dtype, shape, offsets, then the data."""
    import json
    import struct

    (folder / "config.json").write_text(json.dumps(cfg))
    header, blobs, at = {}, [], 0
    for name, t in wt.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hb = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(hb)) + hb + b"".join(blobs))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_command_reads_a_checkpoint_folder_and_writes_the_logits_asked_for(tmp_path, dtype):
    import json
    import os
    import subprocess
    import sys

    cfg = model_cfg([att(mlp=moe(3, 3, 20)), mamba(norm_groups=2, mlp=moe(6, 2, 16)), mamba(heads=2, groups=1, conv=4), att(heads=2, kv=2, dim=16, dims=16)],
                    width=64, vocab=80, loop=(1, 3, 2))
    wt = R.random_checkpoint(cfg, 31)
    write_checkpoint(tmp_path, cfg, wt)
    reqs = {"a": tokens(50, 80, seed=1), "b": tokens(21, 80, seed=2), "c": tokens(70, 80, seed=3)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": reqs["a"][:30], "want": [0, 29]}, {"id": "b", "tokens": reqs["b"][:20], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": reqs["a"][30:31], "want": [0]}, {"id": "b", "tokens": reqs["b"][20:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "c", "tokens": reqs["c"][:64], "want": [5, 63]}], "end": []},       # a sits this step out
             {"step": 3, "entries": [{"id": "a", "tokens": reqs["a"][31:], "want": [18]}, {"id": "c", "tokens": reqs["c"][64:], "want": [0, 5]}],
              "end": ["a", "c"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "192"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True,
                       timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    full = {k: R.forward(cfg, wt, v) for k, v in reqs.items()}
    want = {0: full["a"][[0, 29]], 1: torch.stack([full["a"][30], full["b"][20]]), 2: full["c"][[5, 63]],
            3: torch.stack([full["a"][49], full["c"][64], full["c"][69]])}
    for i, w in want.items():
        got = np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, 80)
        assert got.shape == tuple(w.shape) and close(got, w, dtype, cfg), (i, dtype, rel(got, w))

"""The Sutosun family on the GPU against the float64 reference (oracle/sutosun_ref.py): the engine (scheduler, pages, state
slots, runner, kernels) on small random models (whole prompts, token-by-token decoding, portions down to two tokens, mixed
batches, reuse of pages and slots, greedy generation through the ordinary entry point), models built so that a lost far key, a
lost state, a sink that is left out or a query factor that steps one token late shows, and kernels alone."""
import math

import numpy as np
import pytest
import torch

from oracle import sutosun_ref as R

pytestmark = pytest.mark.gpu
F64 = torch.float64
DEV = "cuda:0"


# ---- small models ------------------------------------------------------------------------------------------------------

def att(heads=6, kv=2, dim=12, vdim=10, scale=0.3, coef=0.4, every=7, mlp=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv, "vdim": vdim, "scale": scale}
    if coef is not None:
        m["q_temp"] = {"coef": coef, "every": every}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def ret(heads=3, dim=8, vdim=14, dims=None, base=100.0, decay=None, mlp=None):
    m = {"decay": decay if decay is not None else [1.0 - 0.6 * 0.15 ** h for h in range(heads)], "dim": dim, "heads": heads, "vdim": vdim}
    if dims != 0:
        m["rot"] = {"base": base, "dims": dim if dims is None else dims}
    return {"type": "retention", "mixer": m, "mlp": mlp}


def lat(heads=4, dim=6, vdim=10, rank=14, rot_dim=4, base=100.0, scaling="default", scale=0.3, mlp=None):
    m = {"dim": dim, "heads": heads, "vdim": vdim, "kv_rank": rank, "rot_dim": rot_dim, "scale": scale}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim}
        if scaling == "default":
            m["rot"]["scaling"] = {"factor": 3.0, "original": 40, "fast": 4.0, "slow": 0.5}
        elif scaling is not None:
            m["rot"]["scaling"] = scaling
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=3, ff=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model_cfg(layers, width=64, vocab=96, cap=9.0, eps=1e-5):
    return {"architecture": "Sutosun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": layers}


def again(layers, j):
    return dict(layers[j], weights_of=j)


def mixed_model(width=64):
    """Every mixer, both feed-forwards, a layer without one, layers that run another layer's tensors (each kind once)."""
    ls = [ret(mlp=dense()), lat(mlp=moe()), att(mlp=moe(4, 1, 16)), ret(heads=2, dim=10, vdim=6, dims=4)]
    ls += [again(ls, 2), again(ls, 0), att(heads=2, kv=2, dim=8, vdim=20, coef=None, mlp=dense(40)), again(ls, 1)]
    return model_cfg(ls, width=width)


def tc_model(experts=True):
    """Sizes that take the tensor-core kernels in bf16: GEMM blocks of 64, latents of 72 + 24 and 64 + 32, the chunked recurrence."""
    f = (lambda: moe(4, 2, 64)) if experts else (lambda: dense(64))
    ls = [ret(heads=2, dim=64, vdim=64, decay=[0.9, 0.995], mlp=dense(128)), lat(heads=4, dim=64, vdim=32, rank=72, rot_dim=24, scale=0.1, mlp=f()),
          att(heads=6, kv=2, dim=64, vdim=48, scale=0.12, coef=0.2, every=64, mlp=f()), ret(heads=3, dim=32, vdim=40, dims=16, decay=[0.5, 0.97, 0.9995]),
          lat(heads=8, dim=32, vdim=64, rank=64, rot_dim=32, scale=0.12, mlp=dense(64))]
    return model_cfg(ls + [again(ls, 0), again(ls, 2)], width=128)


def engine(cfg, wt, dtype="float32", **kw):
    from atx.config import EngineConfig, ModelSource
    from atx.engine import LLMEngine
    from atx.models import sutosun

    mcfg = sutosun.Config.from_json(cfg)
    xt = torch.float32 if dtype == "float32" else torch.bfloat16
    w = sutosun.Weights.from_state_dict(mcfg, wt, torch.device(DEV), xt)
    ecfg = EngineConfig(max_model_len=kw.pop("max_model_len", 256), max_num_seqs=kw.pop("max_num_seqs", 4),
                        max_num_batched_tokens=kw.pop("max_num_batched_tokens", 256),
                        num_gpu_blocks=kw.pop("num_gpu_blocks", 64),
                        enable_prefix_caching=kw.pop("enable_prefix_caching", False),
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


TOL = {"float32": 4e-5, "bfloat16": 0.08}      # bf16: operand rounding through up to eight layers; fp32 is the sharp test


def has_experts(cfg):
    return any((l.get("mlp") or {}).get("kind") == "moe" for l in cfg["layers"])


def close(got, want, dtype, cfg):
    """Every row within the tolerance. One exception: a bf16 model with a mixture of experts. Choosing experts is a
    discontinuous step, so where two router outputs of the reference lie closer than bf16 rounding of the router's input moves
    them, the engine may rightly pick the other one, and that token (and, through the mixers, a few after it) then differs
    by a visible amount. There four rows in five must be within the tolerance and none may be far off. The fp32 runs of the
    same models are held to the sharp limit on every row."""
    rows = rel_rows(got, want)
    if dtype == "bfloat16" and has_experts(cfg):
        return float(rows.quantile(0.8)) < TOL[dtype] and float(rows.max()) < 0.7
    return float(rows.max()) < TOL[dtype]


def whole(eng, rid, toks, end=True):
    return eng.feed([(rid, toks, list(range(len(toks))))], [rid] if end else [])


def in_portions(eng, rid, toks, cuts):
    assert sum(cuts) == len(toks)
    out, at = [], 0
    for n in cuts:
        out.append(eng.feed([(rid, toks[at:at + n], list(range(n)))], [rid] if at + n == len(toks) else []))
        at += n
    return np.concatenate(out)


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
    "attention_no_query_factor": lambda: att(coef=None),
    "attention_factor_steps_every_token": lambda: att(coef=0.7, every=1),
    "attention_factor_steps_at_a_page": lambda: att(coef=1.5, every=16),
    "attention_one_head": lambda: att(heads=1, kv=1, dim=4, vdim=3),
    "attention_a_key_value_head_per_head": lambda: att(heads=4, kv=4, dim=16, vdim=16),
    "retention": lambda: ret(),
    "retention_no_rotation": lambda: ret(dims=0),
    "retention_part_of_the_head_turns": lambda: ret(dim=12, dims=4),
    "retention_one_head_no_decay": lambda: ret(heads=1, dim=8, vdim=8, decay=[1.0]),
    "retention_fast_decay": lambda: ret(heads=2, dim=6, vdim=5, decay=[0.05, 0.3]),
    "retention_key_size_of_the_packed_path": lambda: ret(heads=2, dim=32, vdim=40),
    "retention_wide_keys": lambda: ret(heads=1, dim=72, vdim=8, dims=70),
    "latent": lambda: lat(),
    "latent_unscaled_rotation": lambda: lat(scaling=None),
    "latent_no_rotated_part": lambda: lat(rot_dim=0),
    "latent_every_pair_in_the_stretched_band": lambda: lat(rot_dim=8, base=4.0,
                                                          scaling={"factor": 8.0, "original": 64, "fast": 64.0, "slow": 0.01}),
    "latent_one_head": lambda: lat(heads=1, dim=2, vdim=1, rank=3, rot_dim=2),
    "dense_ffn": lambda: att(heads=2, kv=1, dim=4, vdim=4, mlp=dense(24)),
    "moe": lambda: att(mlp=moe()),
    "moe_one_choice": lambda: ret(mlp=moe(4, 1, 16)),
    "moe_every_expert_chosen": lambda: lat(mlp=moe(3, 3, 16)),
    "tensor_core_sizes": lambda: att(heads=4, kv=2, dim=64, vdim=64, scale=0.125, mlp=moe(4, 2, 64)),
    "tensor_core_dense": lambda: ret(heads=2, dim=64, vdim=64, mlp=dense(128)),
    "between_tile_widths": lambda: lat(heads=2, dim=40, vdim=24, rank=72, rot_dim=24, scale=0.12),
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
    got = in_portions(eng, "b", toks, [1, 2, 61, 1, 1, 2, 80, 1, 1])
    assert close(got, want, dtype, cfg), (kind, width, dtype, rel(got, want))
    eng.runner.close()


def test_first_tokens_of_a_sequence():
    """A zero state, a sink beside one key, a factor of one; one- to four-token prompts."""
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_residual_stream_after_every_layer(dtype):
    cfg = mixed_model() if dtype == "float32" else tc_model(experts=False)
    wt = R.random_checkpoint(cfg, 6)
    for n in (40, 90):        # decode-sized (split-K adds into the stream) and prompt-sized steps
        toks = tokens(n, seed=2)
        eng = engine(cfg, wt, dtype)
        eng.runner.layer_probe = []
        whole(eng, "p", toks)
        got, eng.runner.layer_probe = eng.runner.layer_probe, None
        want = []
        R.forward(cfg, wt, toks, want)
        assert len(got) == len(want) == len(cfg["layers"])
        for i, (g, x) in enumerate(zip(got, want)):
            assert float((g.double().cpu() - x).abs().max()) < (1e-5 if dtype == "float32" else 0.03) * float(x.abs().max()), (n, i)
        eng.runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prefill_token_by_token_and_portions_agree(dtype):
    cfg = mixed_model()
    wt = R.random_checkpoint(cfg, 7)
    toks = tokens(90, seed=3)
    want = R.forward(cfg, wt, toks)
    eng = engine(cfg, wt, dtype)
    a = whole(eng, "w", toks)
    b = in_portions(eng, "t", toks, [1] * 90)
    c = in_portions(eng, "p", toks, [2, 5, 16, 3, 2, 17, 31, 2, 12])         # page borders (16) inside portions
    for name, got in (("whole", a), ("token by token", b), ("portions", c)):
        assert close(got, want, dtype, cfg), (name, dtype, rel(got, want))
    if dtype == "float32":
        assert rel(b, a) < 1e-5 and rel(c, a) < 1e-5
    eng.runner.close()


def test_long_decoding():
    cfg = mixed_model()
    wt = R.random_checkpoint(cfg, 8)
    toks = tokens(200, seed=4)
    want = R.forward(cfg, wt, toks)
    eng = engine(cfg, wt)
    assert rel(in_portions(eng, "d", toks, [9] + [1] * 191), want) < TOL["float32"]
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


def test_bf16_portions_on_the_tensor_cores_beside_single_tokens():
    """Portions (prompt forms of the attention and recurrence kernels) beside single tokens (decode forms, several key
    slices) in one step, portions that start and end inside a 64-token chunk, steps of the query factor inside tiles."""
    cfg = tc_model()
    wt = R.random_checkpoint(cfg, 10)
    reqs = {"a": tokens(230, seed=1), "b": tokens(150, seed=2), "c": tokens(200, seed=3)}
    steps = [[("a", 128), ("b", 2)], [("a", 1), ("b", 100), ("c", 70)], [("a", 1), ("b", 1), ("c", 129)],
             [("a", 100), ("b", 47), ("c", 1)]]
    eng = engine(cfg, wt, "bfloat16", max_model_len=256, max_num_batched_tokens=512, num_gpu_blocks=48)
    got = run_steps(eng, reqs, steps)
    for k, toks in reqs.items():
        assert close(got[k], R.forward(cfg, wt, toks), "bfloat16", cfg), (k, rel(got[k], R.forward(cfg, wt, toks)))
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


def shared_order(order):
    base = [ret(mlp=moe(4, 2, 8)), att(mlp=dense(30)), lat()]
    return model_cfg([dict(base[o], weights_of=order.index(o)) if order.index(o) != i else base[o] for i, o in enumerate(order)])


ODD = {
    "no_cap": lambda: dict(model_cfg([ret(mlp=dense()), att()]), logit_softcap=None),
    "only_recurrent_layers": lambda: model_cfg([ret(), ret(heads=1, dim=5, vdim=3, dims=4, decay=[0.8], mlp=moe())]),
    "no_recurrent_layer": lambda: model_cfg([att(mlp=moe()), lat(mlp=dense())]),
    "tensors_of_a_later_layer": lambda: model_cfg([dict(att(mlp=dense(30)), weights_of=2), ret(), att(mlp=dense(30))]),
    "every_layer_twice_and_more": lambda: shared_order([0, 1, 2, 1, 0, 0, 2, 1]),
    "widths_off_every_block": lambda: model_cfg([ret(heads=3, dim=5, vdim=7, dims=2, mlp=dense(13)), att(heads=3, kv=1, dim=6, vdim=5, mlp=moe(3, 2, 7)),
                                                 lat(heads=3, dim=5, vdim=3, rank=9, rot_dim=2)], width=52, vocab=77),
    "value_wider_than_key": lambda: model_cfg([att(heads=2, kv=1, dim=8, vdim=72, mlp=dense()), ret(heads=2, dim=4, vdim=72)]),
    "latent_wider_than_a_tile": lambda: model_cfg([lat(heads=2, dim=8, vdim=8, rank=264), lat(rank=136, rot_dim=8)]),
    "many_heads_on_one_key_value_head": lambda: model_cfg([att(heads=72, kv=1, dim=8, vdim=8), lat(heads=66, dim=8, vdim=8, rank=16, rot_dim=8)]),
    "many_experts": lambda: model_cfg([att(mlp=moe(40, 6, 8))]),
    "slow_rotation_long_original": lambda: model_cfg([lat(rot_dim=6, base=300000.0, scaling={"factor": 5.0, "original": 2048, "fast": 16.0, "slow": 2.0}),
                                                      ret(dim=16, base=1e6)]),
    "large_eps_small_stream": lambda: model_cfg([ret(mlp=dense()), att(), lat(mlp=moe())], eps=0.3),
}


@pytest.mark.parametrize("name", sorted(ODD))
def test_odd_configurations_whole_and_in_portions(name):
    cfg = ODD[name]()
    wt = R.random_checkpoint(cfg, 14)
    toks = tokens(75, vocab=cfg["vocab"], seed=5)
    want = R.forward(dict(cfg, logit_softcap=cfg["logit_softcap"] or 1e9), wt, toks)
    for dtype in ("float32", "bfloat16"):
        eng = engine(cfg, wt, dtype)
        assert close(whole(eng, "w", toks), want, dtype, cfg), (name, dtype)
        assert close(in_portions(eng, "p", toks, [3, 2, 30, 1, 1, 38]), want, dtype, cfg), (name, dtype)
        eng.runner.close()


def drawn_model(seed):
    g = torch.Generator().manual_seed(seed)

    def ri(lo, hi):
        return int(torch.randint(lo, hi + 1, (1,), generator=g))

    width, layers = 8 * ri(4, 14), []
    for i in range(ri(2, 7)):
        own = [j for j, l in enumerate(layers) if "weights_of" not in l]
        if own and ri(0, 3) == 0:
            layers.append(again(layers, own[ri(0, len(own) - 1)]))
            continue
        mlp = [None, dense(ri(5, 90)), moe(ri(1, 9), 1, ri(4, 40))][ri(0, 2)]
        if mlp and mlp["kind"] == "moe":
            mlp["router"]["top"] = ri(1, min(4, mlp["router"]["experts"]))
        kind = ri(0, 2)
        if kind == 0:
            h, d = ri(1, 4), ri(2, 40)
            layers.append(ret(heads=h, dim=d, vdim=ri(2, 40), dims=2 * ri(1, d // 2), base=float(ri(10, 10 ** 6)),
                              decay=[1.0 - 0.5 ** ri(1, 12) for _ in range(h)], mlp=mlp))
        elif kind == 1:
            sc = {"factor": float(ri(2, 8)), "original": ri(8, 64), "fast": float(ri(2, 40)), "slow": 0.25 * ri(1, 8)} if ri(0, 1) else None
            layers.append(lat(heads=ri(1, 4), dim=ri(1, 24), vdim=ri(1, 24), rank=ri(2, 40), rot_dim=2 * ri(1, 6), base=float(ri(10, 100000)),
                              scaling=sc, scale=0.05 * ri(1, 10), mlp=mlp))
        else:
            kv = ri(1, 3)
            layers.append(att(heads=kv * ri(1, 3), kv=kv, dim=2 * ri(1, 16), vdim=ri(1, 30), scale=0.05 * ri(1, 10), coef=0.1 * ri(0, 10),
                              every=ri(1, 40), mlp=mlp))
    return model_cfg(layers, width=width, vocab=ri(30, 200), cap=float(ri(2, 40)))


def close_drawn(got, want, dtype, cfg):
    """Drawn models have heads of a few dimensions and experts chosen one of two. A unit norm over a retention head whose output
    nearly cancels amplifies rounding of that row, and one expert choice that bf16 rounding flips moves its row and, through the
    mixers, later ones. So here all but a few rows are held to the tolerance and no row may be off by more than a little (fp32) or
    its own size (bf16 with experts); models of fixed sizes are held to it on every row above."""
    rows = rel_rows(got, want)
    if dtype == "float32":
        return float(rows.quantile(0.9)) < TOL[dtype] and float(rows.max()) < 3e-4
    if has_experts(cfg):
        return float(rows.median()) < TOL[dtype] and float(rows.max()) < 1.5
    return float(rows.quantile(0.97)) < TOL[dtype] and float(rows.max()) < 0.6


@pytest.mark.parametrize("draw", range(8))
def test_drawn_models_whole_cut_and_mixed(draw):
    cfg = drawn_model(100 + draw)
    wt = R.random_checkpoint(cfg, 200 + draw)
    V = cfg["vocab"]
    reqs = {"a": tokens(80, V, seed=1), "b": tokens(47, V, seed=2), "c": tokens(9, V, seed=3)}
    want = {k: R.forward(cfg, wt, v) for k, v in reqs.items()}
    steps = [[("a", 17), ("c", 2)], [("a", 1), ("b", 31), ("c", 1)], [("a", 2), ("b", 1), ("c", 1)], [("a", 60), ("b", 15), ("c", 5)]]
    for dtype in ("float32", "bfloat16"):
        eng = engine(cfg, wt, dtype)
        alone = np.concatenate([eng.feed([(k, v, list(range(len(v))))], [k]) for k, v in reqs.items()])
        assert close_drawn(alone, torch.cat([want[k] for k in reqs]), dtype, cfg), (draw, dtype, cfg)
        got = run_steps(eng, reqs, steps)
        assert close_drawn(np.concatenate([got[k] for k in reqs]), torch.cat([want[k] for k in reqs]), dtype, cfg), (draw, dtype, cfg)
        if dtype == "float32":      # the cut must not matter, whatever the conditioning
            assert rel(np.concatenate([got[k] for k in reqs]), alone) < 1e-4, (draw, cfg)
        eng.runner.close()


# ---- models built so that a fault shows ---------------------------------------------------------------------------------------

def pointed_model(kind, dim=32, turned=False):
    """One layer in which the query of token 0 scores the key of token 1 far above every other key. Embeddings of the two tokens are
    axes of their own; the query row and key row they select have a component that nothing else has. `turned` (latent layers): the
    component lies in the rotated part, so the score depends on the distance."""
    W = 64
    if kind == "attention":
        cfg = model_cfg([att(heads=4, kv=2, dim=dim, vdim=32, scale=14.0 / dim, coef=0.1, every=100)], width=W, cap=40.0)
    else:
        cfg = model_cfg([lat(heads=4, dim=dim, vdim=32, rank=40, rot_dim=16, base=30.0, scale=0.3)], width=W, cap=40.0)
    wt = R.random_checkpoint(cfg, 19)
    E = torch.randn(96, W, generator=torch.Generator().manual_seed(4), dtype=F64)
    E[:, :2] = 0.0
    E[0], E[1] = 0.0, 0.0
    E[0, 0] = E[1, 1] = W ** 0.5
    wt["embed"] = E
    for n in ("embed.norm", "l0.norm1"):
        wt[n] = torch.ones(W, dtype=F64)
    q = wt["l0.mix.q"]
    if kind == "attention":
        k = wt["l0.mix.k"]
        q[::dim], k[::dim] = 0.0, 0.0                 # the first row of every head ...
        q[:, 0], k[:, 1] = 0.0, 0.0
        q[::dim, 0], k[::dim, 1] = 1.0, 1.0           # ... answers to one of the two tokens only
        for n in ("q", "k"):
            wt[f"l0.mix.{n}.b"][::dim] = 0.0
            wt[f"l0.mix.{n}.norm"] = torch.ones_like(wt[f"l0.mix.{n}.norm"])
    else:
        D, Rd, C = dim, 16, 40
        row = D if turned else 0                      # row of a head's query that carries the component
        dkv, uk = wt["l0.mix.dkv"], wt["l0.mix.uk"]
        q[row::D + Rd] = 0.0
        q[:, 0] = 0.0
        q[row::D + Rd, 0] = 1.0
        dkv[:, 1] = 0.0
        if turned:
            dkv[C] = 0.0
            dkv[C, 1] = 1.0
            dkv[1, 1] = 1.0                           # (a latent of its own all the same)
        else:
            dkv[0] = 0.0
            dkv[0, 1] = 1.0
            uk[:, 0] = 0.0
            uk[::D] = 0.0
            uk[::D, 0] = 1.0
        wt["l0.mix.dkv.norm"] = torch.ones(C, dtype=F64)
    wt["l0.mix.o"] = wt["l0.mix.o"] * 3.0
    return cfg, {k: t.to(torch.bfloat16).to(F64) for k, t in wt.items()}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
def test_a_far_key_among_hundreds_is_found_at_every_place(kind, dtype):
    """The pointed-at key sits at the first token, on both sides of page borders, at the edges of a prompt portion and in the last
    row in front of the query; the query comes in a prompt and as a decoded token, with several key slices in flight."""
    cfg, wt = pointed_model(kind)
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
    cfg, wt = pointed_model("latent_attention", turned=True)
    eng = engine(cfg, wt, max_logit_rows=16)
    rows = []
    for place in (3, 4, 60, 119):
        toks = [t + 2 if t < 2 else t for t in tokens(120, seed=13)] + [0]
        toks[place] = 1
        want = R.forward(cfg, wt, toks)[-1:]
        eng.feed([("r", toks[:77], [])])
        got = eng.feed([("r", toks[77:], [43])], ["r"])
        assert rel(got, want) < 1e-4, place
        rows.append(want)
    assert rel(rows[2], rows[3]) > 0.02
    eng.runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["attention", "latent_attention"])
def test_the_sink_takes_its_share_unscaled_and_per_head(kind, dtype):
    """Tiny scores and few keys: the sink of head h holds e^s_h / (e^s_h + n) of the weight, from next to nothing to nearly all."""
    layer = att(heads=4, kv=2, dim=64, vdim=64, scale=0.003) if kind == "attention" else lat(heads=4, dim=64, vdim=64, rank=64, rot_dim=32, scale=0.003)
    cfg = model_cfg([layer], width=64)
    wt = R.random_checkpoint(cfg, 24)
    wt["l0.mix.o"] = wt["l0.mix.o"] * 4.0
    wt["l0.mix.sink"] = torch.tensor([-20.0, 0.0, 1.5, 4.0], dtype=F64)
    toks = tokens(6, seed=5)
    want = R.forward(cfg, wt, toks)
    shift = R.forward(cfg, dict(wt, **{"l0.mix.sink": wt["l0.mix.sink"].roll(1)}), toks)
    assert rel(shift, want) > 0.1                                         # a sink of the wrong head shows
    eng = engine(cfg, wt, dtype)
    tol = TOL["float32"] if dtype == "float32" else 0.03
    assert rel(whole(eng, "w", toks), want) < tol
    assert rel(in_portions(eng, "d", toks, [2, 1, 1, 2]), want) < tol
    eng.runner.close()


def test_the_query_factor_steps_at_its_token():
    """Sharp scores and a large coefficient: a factor that steps a token early or late replaces the rows at the step."""
    cfg = model_cfg([att(heads=2, kv=1, dim=16, vdim=16, scale=0.6, coef=4.0, every=13), att(heads=2, kv=2, dim=16, vdim=16, scale=0.6, coef=2.0, every=32)])
    wt = R.random_checkpoint(cfg, 25)
    toks = tokens(120, seed=6)
    want = R.forward(cfg, wt, toks)
    late = [dict(l, mixer=dict(l["mixer"], q_temp=dict(l["mixer"]["q_temp"], every=l["mixer"]["q_temp"]["every"] + 1))) for l in cfg["layers"]]
    assert float(rel_rows(R.forward(dict(cfg, layers=late), wt, toks), want)[[12, 31, 63]].min()) > 5e-3
    eng = engine(cfg, wt)
    assert rel(whole(eng, "w", toks), want) < 2e-4
    assert rel(in_portions(eng, "p", toks, [11, 1, 1, 2, 15, 2, 31, 1, 1, 55]), want) < 2e-4
    eng.runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sharp_attention_shows_a_key_that_is_wrongly_seen_or_hidden(dtype):
    """A large score scale makes every soft-max nearly an arg-max over the visible keys, so a key that is wrongly seen or hidden at
    a page border or a portion's start replaces a row's output instead of nudging it."""
    cfg = model_cfg([att(heads=2, kv=1, dim=8, vdim=8, scale=4.0, coef=None), lat(heads=2, dim=8, vdim=8, rank=16, rot_dim=8, scale=4.0)])
    wt = R.random_checkpoint(cfg, 21)
    toks = tokens(140, seed=6)
    want = R.forward(cfg, wt, toks)
    eng = engine(cfg, wt, dtype)
    for got in (whole(eng, "w", toks), in_portions(eng, "p", toks, [15, 2, 16, 1, 1, 33, 17, 2, 53])):
        if dtype == "float32":
            assert rel(got, want) < 5e-4     # sharp scores amplify fp32 rounding; a fault is of order 1
        else:       # bf16 moves near-ties of a sharp soft-max; a fault of the mask would move most rows by their whole size
            assert float(rel_rows(got, want).quantile(0.7)) < 0.15
    eng.runner.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_state_that_barely_decays_carries_far_tokens_across_steps_and_slots(dtype):
    cfg = model_cfg([ret(heads=2, dim=8, vdim=8, decay=[0.9999, 1.0]), ret(heads=1, dim=32, vdim=16, decay=[0.9995], base=1e5, mlp=dense())])
    wt = R.random_checkpoint(cfg, 22)
    a, b = tokens(230, seed=7), tokens(190, seed=8)
    wa, wb = R.forward(cfg, wt, a), R.forward(cfg, wt, b)
    other = R.forward(cfg, wt, tokens(100, seed=70) + a[100:])             # the reference itself: the last rows depend on the first hundred
    assert rel(other[-10:], wa[-10:]) > 0.2
    eng = engine(cfg, wt, dtype, max_num_seqs=2)
    got = run_steps(eng, {"a": a, "b": b}, [[("a", 64), ("b", 3)], [("a", 65), ("b", 1)], [("a", 1), ("b", 128)],
                                            [("a", 1), ("b", 1)], [("a", 99), ("b", 57)]])
    assert close(got["a"], wa, dtype, cfg) and close(got["b"], wb, dtype, cfg), (rel(got["a"], wa), rel(got["b"], wb))
    # the slots again, from position 0: the old states must be gone
    got = run_steps(eng, {"c": b[:40], "d": a[:50]}, [[("c", 40), ("d", 2)], [("d", 48)]])
    assert close(got["c"], wb[:40], dtype, cfg) and close(got["d"], wa[:50], dtype, cfg)
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
    from atx.scheduler import SamplingParams

    cfg = tc_model(experts=False)      # a choice between experts that bf16 rounding flips would move whole rows
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


def test_without_a_recurrent_layer_cached_prefixes_are_attached():
    """Attention layers alone keep nothing outside the pages: no state slots, and a repeated prompt reads its cached pages."""
    from atx.scheduler import SamplingParams

    cfg = model_cfg([att(mlp=dense()), lat(mlp=moe())])
    wt = R.random_checkpoint(cfg, 18)
    eng = engine(cfg, wt, enable_prefix_caching=True)
    assert eng.state_slots is None
    p = tokens(70, seed=4)
    first = eng.generate_sync([p], SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    second = eng.generate_sync([p + first[0][:3]], SamplingParams(temperature=0.0, max_tokens=3, ignore_eos=True))
    assert second[0] == first[0][3:]
    eng.runner.close()


def test_named_shape_generates_through_the_registry():
    from atx.config import EngineConfig, resolve_model
    from atx.engine import LLMEngine
    from atx.scheduler import SamplingParams

    src = resolve_model("random:sutosun-tiny:3")
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
    i32 = torch.int32
    return (dev(starts, i32), dev(np.asarray(counts, np.int32), i32), dev(np.asarray(pos0, np.int32), i32), dev(np.asarray(slots, np.int32), i32))


@pytest.mark.parametrize("H,D,V,rd,pad", [(2, 64, 128, 64, 0), (1, 32, 40, 16, 0), (3, 96, 130, 96, 2), (2, 128, 16, 64, 0), (2, 64, 64, 12, 1),
                                          (1, 32, 64, 0, 0), (2, 10, 7, 6, 3), (1, 288, 16, 288, 0)])
def test_rotated_recurrence_both_forms_against_the_sum_over_pairs(H, D, V, rd, pad):
    """Two sequences advance through several steps, changing between the token-by-token and the chunked form from the same slot (where
    the key size has the second); a head that keeps everything beside one that forgets within a few tokens."""
    from atx.models.common import rotation_table

    L, _ = lib()
    g = torch.Generator().manual_seed(D + V)
    bf = lambda t: t.to(torch.bfloat16).float()
    n, kmul, base = {"a": 150, "b": 37}, 0.3, 50.0
    chunk_ok = bool(L.atx_linear_recurrence_chunked_supported(D))
    decay = torch.tensor([[1.0, 0.6, 0.98][h % 3] for h in range(H)])
    data, want = {}, {}
    fr, _ = R.pair_frequencies(rd, base) if rd else (None, 1.0)
    for k_, nn in n.items():
        q, k, v = (torch.randn(nn, H * m, generator=g) for m in (D, D, V))
        v = bf(v)
        data[k_] = (q, k, v)
        qq, kk = q.double().view(nn, H, D), k.double().view(nn, H, D)
        if rd:
            qq, kk = R.rotate_halves(qq, fr), R.rotate_halves(kk, fr)
        want[k_] = torch.cat([R.decayed_pair_sum(qq[:, h], kk[:, h] * kmul, v[:, h * V:(h + 1) * V].double(), float(decay[h])) for h in range(H)], 1)
    table = rotation_table(base, rd, 160, torch.device(DEV)) if rd else None
    tp = table.data_ptr() if rd else None
    dd = dev(decay.float())
    state = torch.full((3, H, D, V), 55.0, dtype=torch.float32, device=DEV)
    at, got, used = {"a": 0, "b": 0}, {"a": [], "b": []}, set()
    for na, nb, chunked in [(33, 3, True), (1, 2, False), (16, 31, True), (100, 1, True)]:
        live = [(k_, c, s) for k_, c, s in (("b", nb, 0), ("a", na, 2)) if c > 0 and at[k_] < n[k_]]
        rows = [torch.cat([data[k_][j][at[k_]:at[k_] + c] for k_, c, _ in live]) for j in range(3)]
        starts, cnt, pos0, slots = seq_view([c for _, c, _ in live], [at[k_] for k_, _, _ in live], [s for *_, s in live])
        T = rows[0].shape[0]
        src = torch.zeros(T, 2 * H * D + H * V + pad, device=DEV)        # one fused projection row, possibly off every alignment
        src[:, pad:] = torch.cat(rows, 1).to(DEV)
        p, ld = src.data_ptr() + 4 * pad, src.shape[1]
        y = torch.zeros(T, H * V, dtype=torch.float32, device=DEV)
        use = chunked and chunk_ok
        used.add(use)
        fn = L.atx_linear_recurrence_rot_chunked if use else L.atx_linear_recurrence_rot
        ck(fn(p, ld, p + 4 * H * D, ld, p + 8 * H * D, ld, H, H, D, V, dd.data_ptr(), None, None, None, 0, tp, rd, kmul, state.data_ptr(),
              y.data_ptr(), H * V, starts.data_ptr(), cnt.data_ptr(), pos0.data_ptr(), slots.data_ptr(), len(live), 0, stream()))
        torch.cuda.synchronize()
        o = 0
        for k_, c, _ in live:
            got[k_].append(y[o:o + c].double().cpu())
            o += c
            at[k_] += c
    for k_ in n:
        res = torch.cat(got[k_])
        assert res.shape == want[k_].shape and bool(torch.isfinite(res).all())
        for h in range(H):      # head by head: the one that keeps everything is much larger than the one that forgets
            r, w = res[:, h * V:(h + 1) * V], want[k_][:, h * V:(h + 1) * V]
            err = (r - w).abs().amax(-1) / w.abs().amax(-1).clamp(min=0.2 * float(w.abs().max()))
            assert float(err.max()) < (0.03 if True in used else 3e-5), (k_, h, float(err.max()))


def test_recurrence_refuses_what_it_does_not_have():
    L, _ = lib()
    x = torch.zeros(64, device=DEV)
    i = torch.zeros(4, dtype=torch.int32, device=DEV)
    p, ip = x.data_ptr(), i.data_ptr()
    for fn in (L.atx_linear_recurrence_rot, L.atx_linear_recurrence_rot_chunked):
        for rd, act, table in ((3, 0, p), (34, 0, p), (8, 1, p), (8, 0, None)):
            assert fn(p, 32, p, 32, p, 32, 1, 1, 32, 1, p, None, None, None, act, table, rd, 1.0, p, p, 1, ip, ip, ip, ip, 1, 0, stream()) != 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,V", [(6, 2, 12, 10), (4, 4, 64, 48), (3, 1, 6, 5)])
def test_query_and_key_preparation_with_a_growing_query_factor(H, G, D, V, dtype):
    L, Cb = lib()
    xt, dt = types(dtype)
    g = torch.Generator().manual_seed(H + D)
    every, coef, eps, bs = 16.0, 0.8, 1e-5, 16
    pos = np.array([0, 14, 15, 16, 30, 31, 32, 1000, 4095, 65534, 65535, 131071], np.int32)
    T, ld = len(pos), (H + G) * D + G * V + 3
    proj = torch.randn(T, ld, generator=g).float()
    b = {k: (0.5 * torch.randn(m, generator=g)).to(xt) for k, m in (("q", H * D), ("k", G * D), ("v", G * V))}
    w = {k: (1 + 0.2 * torch.randn(m, generator=g)).to(xt) for k, m in (("q", H * D), ("k", G * D))}
    q = torch.zeros(T, H * D, dtype=xt, device=DEV)
    kc, vc = (torch.full((2, G, bs, m), 7.0, dtype=xt, device=DEV) for m in (D, V))
    slots = np.array([5, 31, 0, 1, 2, 3, 4, 16, 17, 18, 19, -1], np.int32)
    pd, bd, wd, posd, sd = dev(proj), {k: dev(t) for k, t in b.items()}, {k: dev(t) for k, t in w.items()}, dev(pos), dev(slots)
    ck(L.atx_qk_prepare_temp(pd.data_ptr(), ld, 0, H * D, (H + G) * D, bd["q"].data_ptr(), bd["k"].data_ptr(), bd["v"].data_ptr(),
                             wd["q"].data_ptr(), wd["k"].data_ptr(), None, 0, coef, every, posd.data_ptr(), sd.data_ptr(), q.data_ptr(),
                             kc.data_ptr(), vc.data_ptr(), T, H, G, D, V, bs, eps, dt, 0, stream()))
    torch.cuda.synchronize()
    x = proj.double()
    f = torch.tensor([1 + coef * math.log(math.floor((p + 1) / every) + 1) for p in pos.tolist()], dtype=F64)
    wq = R.unit_rms(x[:, :H * D] + b["q"].double(), eps) * w["q"].double() * f[:, None]
    wk = R.unit_rms(x[:, H * D:(H + G) * D] + b["k"].double(), eps) * w["k"].double()
    wv = x[:, (H + G) * D:(H + G) * D + G * V] + b["v"].double()
    tol = 2e-6 if dtype == "float32" else 5e-3
    assert float((q.double().cpu()[:-1] - wq[:-1]).abs().max()) < tol * float(wq.abs().max())
    assert float(q[-1].float().abs().max()) == 0.0                      # a padded row is left alone
    for t in range(T - 1):
        s = int(slots[t])
        assert float((kc[s // bs, :, s % bs].double().cpu() - wk[t].view(G, D)).abs().max()) < tol * float(wk.abs().max())
        assert float((vc[s // bs, :, s % bs].double().cpu() - wv[t].view(G, V)).abs().max()) < tol * float(wv.abs().max())
    assert float((kc[0, :, 15] - 7.0).abs().max()) == 0.0
    assert L.atx_qk_prepare_temp(pd.data_ptr(), ld, 0, H * D, (H + G) * D, None, None, None, None, None, None, 0, coef, 0.0, posd.data_ptr(),
                                 sd.data_ptr(), q.data_ptr(), kc.data_ptr(), vc.data_ptr(), T, H, G, D, V, bs, eps, dt, 0, stream()) != 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W", [40, 38, 64, 520, 2048, 6000])
def test_the_stream_starts_as_a_normed_embedding_row(W, dtype):
    import ctypes

    L, Cb = lib()
    xt, dt = types(dtype)
    g = torch.Generator().manual_seed(W)
    T, V, eps = 9, 30, 1e-3
    table, tw, w1 = (0.5 * torch.randn(V, W, generator=g)).to(xt), (1 + 0.2 * torch.randn(W, generator=g)).to(xt), (1 + 0.2 * torch.randn(W, generator=g)).to(xt)
    ids = torch.randint(0, V, (T,), generator=g).to(torch.int32)
    h, out = torch.full((T, W), 9.0, device=DEV), torch.zeros(T, W, dtype=xt, device=DEV)
    td, twd, wd, idd = dev(table), dev(tw), dev(w1), dev(ids)
    t = Cb.ResidTerms()
    t.y_scale, t.table_mode, t.ids, t.table, t.table_w, t.vocab = 1.0, Cb.TABLE_START, idd.data_ptr(), td.data_ptr(), twd.data_ptr(), V
    ck(L.atx_parallel_resid_norm(h.data_ptr(), ctypes.byref(t), wd.data_ptr(), out.data_ptr(), None, None, 0.0, None, T, W, eps, None, 0, dt, 0, stream()))
    torch.cuda.synchronize()
    x = R.unit_rms(table.double()[ids.long()], eps) * tw.double()
    assert float((h.double().cpu() - x).abs().max()) < 1e-5
    want = R.unit_rms(x, eps) * w1.double()
    assert float((out.double().cpu() - want).abs().max()) < (1e-5 if dtype == "float32" else 0.01) * float(want.abs().max())
    # the next sublayer's weighted expert outputs join the stream; gathered rows of it go out without being stored
    top = 2
    ye, wgt = torch.randn(T * top, W, generator=g).float(), torch.rand(T, top, generator=g).float()
    sl = torch.randperm(T * top, generator=g).to(torch.int32)
    yd, gd, sd, rows = dev(ye), dev(wgt), dev(sl), dev(torch.tensor([7, 0, 7], dtype=torch.int32))
    t = Cb.ResidTerms()
    t.y_scale, t.experts, t.wgt, t.slot_of, t.lde, t.top = 1.0, yd.data_ptr(), gd.data_ptr(), sd.data_ptr(), W, top
    out2 = torch.zeros(3, W, dtype=xt, device=DEV)
    ck(L.atx_parallel_resid_norm(h.data_ptr(), ctypes.byref(t), wd.data_ptr(), out2.data_ptr(), None, None, 0.0, rows.data_ptr(), 3, W, eps, None, 0, dt, 0,
                                 stream()))
    torch.cuda.synchronize()
    assert float((h.double().cpu() - x).abs().max()) < 1e-5
    full = x + (wgt.double()[:, :, None] * ye.double()[sl.long().view(T, top)]).sum(1)
    want2 = (R.unit_rms(full, eps) * w1.double())[[7, 0, 7]]
    assert float((out2.double().cpu() - want2).abs().max()) < (1e-5 if dtype == "float32" else 0.01) * float(want2.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_gelu_gate_and_unit_norm_per_head_without_weights(dtype):
    L, Cb = lib()
    xt, dt = types(dtype)
    tol = 1e-5 if dtype == "float32" else 0.01
    g = torch.Generator().manual_seed(3)
    T, I = 7, 37
    gu = (torch.randn(T, 2 * I, generator=g) * 4).float()
    gu[0, :4] = torch.tensor([-30.0, 30.0, 0.0, -1e-4])
    out, gud = torch.zeros(T, I, dtype=xt, device=DEV), dev(gu)
    for kind, f in ((Cb.ACT_GELU_TANH, R.gelu_tanh), (Cb.ACT_SILU, R.silu)):
        ck(L.atx_gated_act_kind(gud.data_ptr(), out.data_ptr(), T, I, kind, dt, 0, stream()))
        torch.cuda.synchronize()
        want = f(gu[:, :I].double()) * gu[:, I:].double()
        assert float((out.double().cpu() - want).abs().max()) < tol * float(want.abs().max()), kind
    assert L.atx_gated_act_kind(gud.data_ptr(), out.data_ptr(), T, I, Cb.ACT_RELU2, dt, 0, stream()) != 0
    for Hh, Vd in ((3, 10), (2, 64), (9, 128), (2, 260), (1, 7)):
        y, gate = torch.randn(T, Hh * Vd + 4, generator=g).float(), torch.randn(T, Hh * Vd + 4, generator=g).float()
        out, yd, gd = torch.zeros(T, Hh * Vd, dtype=xt, device=DEV), dev(y), dev(gate)
        ck(L.atx_gated_norm_groups(yd.data_ptr(), Hh * Vd + 4, gd.data_ptr(), Hh * Vd + 4, None, 0, out.data_ptr(), Hh * Vd, T, Hh * Vd, Hh, 1e-2, 2, 1.0,
                                   dt, 0, stream()))
        torch.cuda.synchronize()
        want = R.unit_rms(y[:, :Hh * Vd].double().view(T, Hh, Vd), 1e-2).reshape(T, -1) * R.silu(gate[:, :Hh * Vd].double())
        assert float((out.double().cpu() - want).abs().max()) < tol * float(want.abs().max()), (Hh, Vd)


@pytest.mark.parametrize("T,F,K", [(5, 128, 512), (30, 64, 256), (64, 192, 1024), (100, 384, 128), (300, 512, 320)])
def test_gemm_with_the_gelu_gate_in_its_epilogue(T, F, K):
    """Gate and up rows in blocks of 64; decode-sized steps cut K over a cluster and sum the parts before the gate; prompt-sized
    steps take the persistent kernel."""
    from atx.weights import interleave_gate_up

    L, Cb = lib()
    g = torch.Generator().manual_seed(T + F)
    gate, up = ((3.0 * torch.randn(F, K, generator=g) / K ** 0.5).to(torch.bfloat16) for _ in range(2))
    w = interleave_gate_up(gate, up).contiguous().to(DEV)
    x = torch.zeros(max(T, 16), K, dtype=torch.bfloat16, device=DEV)
    x[:T] = torch.randn(T, K, generator=g).to(torch.bfloat16).to(DEV)
    plan = Cb.GemmPlan(w, x)
    out = torch.full((T, F + 8), 3.0, dtype=torch.bfloat16, device=DEV)
    plan.run(out, T, Cb.GEMM_GEGLU_BF16)
    torch.cuda.synchronize()
    xg, xu = x[:T].cpu().double() @ gate.double().T, x[:T].cpu().double() @ up.double().T
    assert torch.allclose(out[:, :F].cpu().double(), R.gelu_tanh(xg) * xu, atol=2e-2, rtol=1e-2)
    assert float((R.gelu_tanh(xg) * xu - R.silu(xg) * xu).abs().max()) > 0.3          # the other gate would show
    assert float((out[:, F:].float() - 3.0).abs().max()) == 0.0


def test_router_bias_moves_choices_and_weights():
    """Both launches (decode-sized steps route and plan in one): the bias is part of the logits, the weights are the soft-max over
    the chosen outputs alone, also where the logits are far apart."""
    L, Cb = lib()
    g = torch.Generator().manual_seed(2)
    T, E = 33, 37
    z, bias = (torch.randn(T, 40, generator=g) * 3).float(), (torch.randn(E, generator=g) * 2).float()
    z[0] *= 20.0
    zd, bd = dev(z), dev(bias)
    i32 = lambda n: torch.full((n,), -7, dtype=torch.int32, device=DEV)
    for top in (1, 4, 37):
        zz = z[:, :E].double() + bias.double()
        val, idx = zz.topk(top, -1)
        want = torch.softmax(val, -1)
        for fused in (False, True):
            sel, wgt = i32(T * top), torch.zeros(T, top, device=DEV)
            if fused:
                so, pm, sl, tl = i32(E + 1), i32(T * top), i32(T * top), i32(2 + 2 * (T * top + E))
                ck(L.atx_moe_route_plan_biased(zd.data_ptr(), 40, bd.data_ptr(), None, E, top, 1.0, 1, Cb.MOE_SOFTMAX, 1, T, E, 64, sel.data_ptr(),
                                               wgt.data_ptr(), so.data_ptr(), pm.data_ptr(), sl.data_ptr(), tl.data_ptr(), 0, stream()))
            else:
                ck(L.atx_moe_route_biased(zd.data_ptr(), 40, bd.data_ptr(), None, E, top, 1.0, 1, Cb.MOE_SOFTMAX, 1, sel.data_ptr(), wgt.data_ptr(), T, 0,
                                          stream()))
            torch.cuda.synchronize()
            got = sel.cpu().long().view(T, top)
            assert torch.equal(got.sort(-1).values, idx.sort(-1).values), (top, fused)
            assert torch.equal(got[1:], idx[1:])      # (row 0's smallest soft-max scores are all zero in fp32: any order)
            assert float((wgt.double().cpu() - want).abs().max()) < 1e-6
            if fused:
                assert int(so[E]) == T * top and sorted(sl.cpu().tolist()) == list(range(T * top))


@pytest.mark.parametrize("T", [1, 3, 16, 17, 50, 64, 90, 700])
def test_silu_experts_decode_tiles_and_the_grouped_gemm(T):
    """The helper the program uses, both dtypes and every path: by-slot outputs summed with their weights, against the definition."""
    from atx.models.common import Experts, gate_up_matrix

    L, Cb = lib()
    for E, top, F, W in ((5, 2, 64, 128), (3, 3, 192, 64), (9, 1, 40, 72), (160, 2, 320, 64), (2, 1, 512, 1024)):
        g = torch.Generator().manual_seed(T + E)
        wt = {f"e{e}.{n}": (torch.randn(*s, generator=g, dtype=F64) * s[1] ** -0.5).to(torch.bfloat16).to(F64)
              for e in range(E) for n, s in (("gate", (F, W)), ("up", (F, W)), ("down", (W, F)))}
        wt["router"], wt["router.b"] = torch.randn(E, W, generator=g, dtype=F64) * 0.3, torch.randn(E, generator=g, dtype=F64)
        x = torch.randn(T, W, generator=g, dtype=F64).to(torch.bfloat16).to(F64)
        want = R.expert_mixture(x, {"router": {"top": top}}, wt, "")
        logits, bias = dev((x @ wt["router"].T).float()), dev(wt["router.b"].float())
        for dtype in ("float32", "bfloat16"):
            xt, dt = types(dtype)
            xn = torch.zeros(max(T, 16), W, dtype=xt, device=DEV)
            xn[:T] = x.to(xt)
            ex = Experts(L, ck, [{"router": {"top": top, "experts": E}, "expert": {"ff": F}}], max(T, 16), W, xn, dt, gated=True,
                         score=Cb.MOE_SOFTMAX, normalize=1)
            up = torch.stack([gate_up_matrix(wt[f"e{e}.gate"], wt[f"e{e}.up"], W, xt)[0] for e in range(E)]).to(device=DEV, dtype=xt).contiguous()
            down = torch.stack([wt[f"e{e}.down"] for e in range(E)]).to(device=DEV, dtype=xt).contiguous()
            n = ex.run(logits.data_ptr(), E, top, up, down, ex.plans(up, down), T, T <= 64, 0, stream(), bias=bias.data_ptr())
            torch.cuda.synchronize()
            assert n == (3 if T <= 64 else 5 if dtype == "bfloat16" and W % 64 == 0 and F % 64 == 0 else 4)
            out = ex.out.view(-1, W).double().cpu()
            sl, wg = ex.slot_of[:T * top].long().cpu().view(T, top), ex.wgt[:T * top].double().cpu().view(T, top)
            assert sorted(sl.flatten().tolist()) == list(range(T * top))
            got = (wg[:, :, None] * out[sl]).sum(1)
            assert float((got - want).abs().max()) < (1e-4 if dtype == "float32" else 0.03) * float(want.abs().max()), (E, dtype)


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

    ls = [att(mlp=moe(3, 3, 20)), ret(mlp=moe(6, 2, 16)), lat(mlp=dense(50)), ret(heads=1, dim=16, vdim=24, decay=[0.97])]
    cfg = model_cfg(ls + [again(ls, 1), again(ls, 0)], width=64, vocab=80)
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

"""Host side of the Lifuzen family: configuration and registry, checkpoint names, the weight layout the kernels read, the order
of execution with a looped block, explicit step plans with state slots, and the reference against itself (scan = sum over
pairs, sink, values = convolved keys, weighted input of an expert = squared weight on its output, pass vectors). No GPU."""
import json

import pytest
import torch

from oracle import lifuzen_ref as R

F64 = torch.float64


def small_cfg(**over):
    moe = {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "top": 2}}
    cfg = {
        "architecture": "Lifuzen", "vocab": 90, "width": 48, "norm": {"eps": 1e-5}, "residual_mult": 0.6, "logit_softcap": 12.0,
        "loop": {"start": 1, "stop": 3, "times": 3},
        "layers": [
            {"type": "mamba2", "mlp": moe,
             "mixer": {"conv": 3, "groups": 2, "heads": 4, "norm_groups": 4, "state": 6, "vdim": 10}},
            {"type": "attention", "mlp": None,
             "mixer": {"conv": 4, "dim": 12, "heads": 6, "kv_heads": 2, "vdim": 12, "rot": {"base": 100.0, "dims": 8}, "scale": 0.3}},
            {"type": "mamba2", "mlp": dict(moe, router={"experts": 3, "top": 3}),
             "mixer": {"conv": 2, "groups": 1, "heads": 3, "norm_groups": 1, "state": 5, "vdim": 8}},
            {"type": "attention", "mlp": moe,
             "mixer": {"conv": 2, "dim": 10, "heads": 2, "kv_heads": 1, "vdim": 10, "rot": {"base": 50.0, "dims": 10}, "scale": 0.2}},
        ],
    }
    cfg.update(over)
    return cfg


def test_config_is_read_from_json_and_picked_by_architecture(tmp_path):
    from atx.config import model_config_from_json, resolve_model
    from atx.models import lifuzen

    cfg = small_cfg()
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    m = model_config_from_json(tmp_path / "config.json")
    assert isinstance(m, lifuzen.Config) and m.architecture == "Lifuzen" and m.recurrent
    assert (m.vocab_size, m.width, m.eps, m.residual_mult, m.logit_softcap) == (90, 48, 1e-5, 0.6, 12.0)
    assert m.runs() == [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (1, 2), (2, 2), (3, None)] == R.execution_order(cfg)
    assert m.num_hidden_layers == 8
    assert resolve_model(str(tmp_path)).config.tensor_shapes() == m.tensor_shapes()
    # every pass of a looped layer has pages and states of its own
    assert m.kv_bytes_per_token(2) == 2 * 2 * (3 * 2 * 12 + 10)
    conv = 2 * (40 + 24) + 3 * 3 * (8 * 12) + 3 * 1 * (24 + 10) + 1 * (3 * 10)
    assert m.state_bytes_per_sequence() == 4 * (conv + 4 * 6 * 10 + 3 * 3 * 5 * 8)
    for path, value in ((("layers", 0, "type"), "gla"), (("layers", 1, "mixer", "kv_heads"), 4), (("layers", 1, "mixer", "vdim"), 8),
                        (("layers", 1, "mixer", "rot", "dims"), 14), (("layers", 1, "mixer", "rot", "dims"), 5),
                        (("layers", 0, "mixer", "groups"), 3), (("layers", 0, "mixer", "norm_groups"), 7),
                        (("layers", 0, "mixer", "conv"), 0), (("layers", 0, "mlp", "router", "top"), 6),
                        (("layers", 0, "mlp", "kind"), "dense"), (("loop", "stop"), 5), (("loop", "times"), 0),
                        (("loop", "start"), 3), (("logit_softcap",), -1.0)):
        bad = json.loads(json.dumps(cfg))
        d = bad
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ValueError):
            lifuzen.Config.from_json(bad)
    plain = json.loads(json.dumps(cfg))           # what a configuration leaves out does not exist
    del plain["loop"], plain["logit_softcap"], plain["residual_mult"], plain["layers"][1]["mixer"]["rot"]
    mp = lifuzen.Config.from_json(plain)
    assert mp.loop is None and mp.logit_softcap == 0.0 and mp.residual_mult == 1.0 and mp.num_hidden_layers == 4
    assert "loop.step" not in mp.tensor_shapes()


def test_checkpoint_names_and_shapes_match_the_reference_listing():
    from atx.models import lifuzen

    cfg = small_cfg()
    assert lifuzen.Config.from_json(cfg).tensor_shapes() == R.checkpoint_shapes(cfg)
    names = R.checkpoint_shapes(cfg)
    assert names["loop.step"] == (3, 48) and "l1.norm2" not in names and "l1.mlp.router" not in names and "head" not in names
    assert names["l1.mix.k.conv"] == (24, 4) and "l1.mix.v" not in names and names["l2.mlp.e2.up"] == (24, 48)
    assert names["l0.mix.in"] == (40 + 40 + 24 + 4, 48) and names["l0.mix.conv"] == (64, 3)


def test_weights_are_stacked_the_way_the_kernels_read_them():
    from atx.models import lifuzen

    cfg = small_cfg()
    wt = R.random_checkpoint(cfg, 1)
    m = lifuzen.Config.from_json(cfg)
    w = lifuzen.Weights.from_state_dict(m, wt, torch.device("cpu"), torch.float32)
    l0, l1, l2, l3 = w.layers
    assert l1.w_in.shape == (72 + 24, 48) and torch.equal(l1.w_in[72:].double(), wt["l1.mix.k"])
    assert l1.conv.shape == (96, 4) and torch.equal(l1.conv[:72].double(), wt["l1.mix.q.conv"]) and l1.norm2 is None
    assert l0.w_up.shape == (5, 24, 48) and torch.equal(l0.w_up[3].double(), wt["l0.mlp.e3.up"])
    assert l2.w_down.shape == (3, 48, 24) and torch.equal(l2.w_down[1].double(), wt["l2.mlp.e1.down"])
    assert l0.skip.dtype == torch.float32 and torch.equal(w.loop_step.double(), wt["loop.step"])
    assert torch.equal(l3.norm1.double(), wt["l3.norm1"])              # stored as they are: the kernel adds the one in fp32
    sd = dict(wt)
    del sd["l0.mlp.router"]
    with pytest.raises(KeyError):
        lifuzen.Weights.from_state_dict(m, sd, torch.device("cpu"), torch.float32)
    with pytest.raises(ValueError):
        lifuzen.Weights.from_state_dict(m, dict(wt, **{"l0.mix.norm": torch.zeros(41)}), torch.device("cpu"), torch.float32)


def test_named_shapes_come_through_the_registry():
    from atx.config import resolve_model

    for name, layers in (("lifuzen-tiny", 4), ("lifuzen-1b", 16), ("lifuzen-8b", 32)):
        c = resolve_model(f"random:{name}:1").config
        assert c.architecture == "Lifuzen" and c.num_hidden_layers == layers
        assert [l["type"] for l in c.layers[:4]] == ["attention", "mamba2", "mamba2", "attention"]
    assert c.weight_bytes_per_decode_step(2, 8) > c.weight_bytes_per_decode_step(2, 1)     # more tokens reach more experts
    assert c.decode_kv_bytes(2000) == 2000 * c.kv_bytes_per_token()
    looped = type(c)(**dict(vars(c), loop={"start": 0, "stop": 4, "times": 2}))
    per = lambda m: m.weight_bytes_per_decode_step(2, 8) - 2 * m.vocab_size * m.width
    assert abs(per(looped) / per(c) - 36 / 32) < 1e-6                   # a looped layer streams its weights once per pass


def test_explicit_step_plans_take_and_return_state_slots():
    from atx.kv_cache import BlockAllocator, StateSlotPool
    from atx.scheduler import SamplingParams, Scheduler, Sequence

    alloc, slots = BlockAllocator(8, 16, False), StateSlotPool(1)
    sch = Scheduler(alloc, 4, 64, 64, (), state_slots=slots)
    p = SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True)
    a, b = Sequence("a", list(range(40)), p, alloc), Sequence("b", [1, 2, 3], p, alloc)
    sch.commit(sch.plan_explicit([(a, 33, [32])]), {})
    with pytest.raises(RuntimeError):
        sch.plan_explicit([(b, 2, [])])
    assert alloc.num_free == 8 - 3
    sch.retire(a)
    plan = sch.plan_explicit([(b, 2, [1])])
    assert len(plan.prefills) == 1 and b.state_slot == 0 and slots.num_free == 0 and alloc.num_free == 7


def test_reference_scan_equals_its_sum_over_pairs():
    g = torch.Generator().manual_seed(0)
    n, H, G, N, P = 11, 4, 2, 3, 5
    x, b, c = (torch.randn(n, *s, generator=g, dtype=F64) for s in ((H, P), (G, N), (G, N)))
    dt, al, d = torch.rand(n, H, generator=g, dtype=F64), torch.randn(H, generator=g, dtype=F64), torch.randn(H, generator=g, dtype=F64)
    got = R.selective_scan(x, b, c, dt, al, d)
    L = torch.cumsum(torch.exp(al) * dt, 0)
    for h in range(H):
        for t in range(n):
            want = d[h] * x[t, h]
            for j in range(t + 1):
                want = want + torch.exp(L[j, h] - L[t, h]) * dt[j, h] * (c[t, h // 2] @ b[j, h // 2]) * x[j, h]
            assert torch.allclose(got[t, h], want)
    assert torch.allclose(R.softplus(torch.tensor([-40.0, 0.0, 40.0], dtype=F64)),
                          torch.tensor([4.248354255291589e-18, 0.6931471805599453, 40.0], dtype=F64))


def test_reference_sink_convolution_rotation_and_expert_weights():
    g = torch.Generator().manual_seed(1)
    # one key: weight e^s / (1 + e^s); a score far below the sink's leaves nothing, far above leaves the value itself
    q = torch.tensor([[[2.0, 0.0]], [[2.0, 0.0]]], dtype=F64)
    k = torch.tensor([[[1.0, 0.0]], [[-50.0, 0.0]]], dtype=F64)
    v = torch.tensor([[[3.0, 1.0]], [[7.0, 7.0]]], dtype=F64)
    o = R.sink_attention(q, k, v, 0.5)
    s = torch.exp(torch.tensor(1.0, dtype=F64))
    assert torch.allclose(o[0, 0], s / (1 + s) * v[0, 0]) and torch.allclose(o[1, 0], s / (1 + s) * v[0, 0])
    assert torch.allclose(R.sink_attention(100 * q, k, v, 0.5)[0, 0], v[0, 0])
    assert float(R.sink_attention(-100 * q, k, v, 0.5)[0].abs().max()) < 1e-20
    # taps: last column = the row itself, zeros in front of the sequence
    u = torch.tensor([[1.0, 2.0], [3.0, 5.0], [7.0, 11.0]], dtype=F64)
    w = torch.tensor([[0.5, 2.0], [0.0, 1.0]], dtype=F64)
    assert R.causal_taps(u, w).tolist() == [[2.0, 2.0], [6.5, 5.0], [15.5, 11.0]]
    assert R.causal_taps(u, w, torch.tensor([1.0, -1.0], dtype=F64))[0].tolist() == [3.0, 1.0]
    # rotation turns adjacent pairs of the first dims elements and keeps their length; position 0 and the rest stay
    x = torch.randn(5, 2, 8, generator=g, dtype=F64)
    y = R.rotate_pairs(x, 6, 50.0)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    assert torch.allclose(y[..., 0::2] ** 2 + y[..., 1::2] ** 2, x[..., 0::2] ** 2 + x[..., 1::2] ** 2)
    assert torch.allclose(y[3, 0, 0], x[3, 0, 0] * torch.cos(torch.tensor(3.0, dtype=F64)) - x[3, 0, 1] * torch.sin(torch.tensor(3.0, dtype=F64)))
    # so the norm over the head may come before or after the rotation
    assert torch.allclose(R.unit_rms(y, 1e-3), R.rotate_pairs(R.unit_rms(x, 1e-3), 6, 50.0))
    # scores are used as they are, and the weight on an expert's input is its square on the output
    wt = {"e.up": torch.randn(9, 4, generator=g, dtype=F64), "e.down": torch.randn(4, 9, generator=g, dtype=F64)}
    h = torch.randn(6, 4, generator=g, dtype=F64)
    assert torch.allclose(R.squared_relu_expert(0.3 * h, wt, "e."), 0.09 * R.squared_relu_expert(h, wt, "e."))
    router = torch.randn(5, 4, generator=g, dtype=F64)
    idx, val = R.route(h, router, 2)
    sc = torch.sigmoid(h @ router.T)
    assert torch.allclose(val, sc.gather(1, idx)) and bool((val.sum(-1) - 1.0).abs().max() > 1e-2)
    assert float(R.soft_cap(torch.tensor(1e6, dtype=F64), 12.0)) == 12.0 and float(R.soft_cap(torch.tensor(5.0, dtype=F64), None)) == 5.0


def test_reference_is_causal_and_every_pass_enters_with_the_embedding_and_its_vector():
    cfg = small_cfg()
    wt = R.random_checkpoint(cfg, 2)
    toks = [int(t) for t in torch.randint(0, 90, (19,), generator=torch.Generator().manual_seed(0))]
    a = R.forward(cfg, wt, toks)
    assert torch.allclose(a[:12], R.forward(cfg, wt, toks[:12])) and a.shape == (19, 90)
    assert float(a.abs().max()) < 12.0
    # silent layers: what is left is the bookkeeping of the passes
    quiet = {k: (torch.zeros_like(t) if k.endswith("mix.o") or k.endswith(".down") else t) for k, t in wt.items()}
    res = []
    R.forward(cfg, quiet, toks, res)
    e, st = wt["embed"][toks], wt["loop.step"]
    assert torch.allclose(res[0], e) and torch.allclose(res[1], e + st[0]) and torch.allclose(res[2], e + st[0])
    assert torch.allclose(res[4], 2 * e + st[0] + st[1]) and torch.allclose(res[7], 3 * e + st[0] + st[1] + st[2])

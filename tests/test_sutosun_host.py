"""Host side of the Sutosun family: configuration and registry, checkpoint names, the weight layout the kernels read, layers that
share tensors, explicit step plans with state slots, and the reference against itself (recurrence = sum over pairs, sink, query
factor, rotation, routing). No GPU."""
import json
import math

import pytest
import torch

from oracle import sutosun_ref as R

F64 = torch.float64


def small_cfg(**over):
    moe = {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 5, "top": 2}}
    att = {"dim": 12, "heads": 6, "kv_heads": 2, "vdim": 10, "scale": 0.3, "q_temp": {"coef": 0.4, "every": 7}}
    cfg = {
        "architecture": "Sutosun", "vocab": 90, "width": 48, "norm": {"eps": 1e-5}, "logit_softcap": 12.0,
        "layers": [
            {"type": "retention", "mlp": moe,
             "mixer": {"decay": [0.5, 0.9, 0.99], "dim": 8, "heads": 3, "vdim": 14, "rot": {"base": 100.0, "dims": 6}}},
            {"type": "attention", "mlp": {"kind": "dense", "ff": 40}, "mixer": att},
            {"type": "latent_attention", "mlp": None,
             "mixer": {"dim": 6, "heads": 4, "vdim": 9, "kv_rank": 20, "rot_dim": 4, "scale": 0.25,
                       "rot": {"base": 50.0, "dims": 4, "scaling": {"factor": 3.0, "original": 40, "fast": 4.0, "slow": 0.5}}}},
            {"type": "attention", "mlp": {"kind": "dense", "ff": 40}, "mixer": att, "weights_of": 1},
        ],
    }
    cfg.update(over)
    return cfg


def test_config_is_read_from_json_and_picked_by_architecture(tmp_path):
    from atx.config import model_config_from_json, resolve_model
    from atx.models import sutosun

    cfg = small_cfg()
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    m = model_config_from_json(tmp_path / "config.json")
    assert isinstance(m, sutosun.Config) and m.architecture == "Sutosun" and m.recurrent
    assert (m.vocab_size, m.width, m.eps, m.logit_softcap, m.num_hidden_layers) == (90, 48, 1e-5, 12.0, 4)
    assert resolve_model(str(tmp_path)).config.tensor_shapes() == m.tensor_shapes()
    # layers that share tensors still have pages and states of their own
    assert m.kv_bytes_per_token(2) == 2 * (2 * 2 * (12 + 10) + 20 + 4)
    assert m.state_bytes_per_sequence() == 4 * 3 * 8 * 14 and m.decode_kv_bytes(100) == 100 * m.kv_bytes_per_token()
    assert not sutosun.Config.from_json(small_cfg(layers=cfg["layers"][1:3])).recurrent
    for path, value in ((("layers", 0, "type"), "gla"), (("layers", 1, "mixer", "kv_heads"), 4), (("layers", 0, "mixer", "rot", "dims"), 5),
                        (("layers", 0, "mixer", "rot", "dims"), 10), (("layers", 0, "mixer", "decay"), [0.5, 0.9]),
                        (("layers", 2, "mixer", "rot", "dims"), 6), (("layers", 2, "mixer", "rot", "dims"), 3),
                        (("layers", 1, "mixer", "q_temp", "every"), 0), (("layers", 0, "mlp", "router", "top"), 6),
                        (("layers", 0, "mlp", "kind"), "sparse"), (("layers", 3, "weights_of"), 3), (("layers", 3, "weights_of"), 4),
                        (("layers", 3, "weights_of"), 0), (("layers", 3, "mixer", "scale"), 0.31), (("logit_softcap",), -1.0)):
        bad = json.loads(json.dumps(cfg))
        d = bad
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(ValueError):
            sutosun.Config.from_json(bad)
    chain = json.loads(json.dumps(small_cfg(layers=cfg["layers"] + [dict(cfg["layers"][3], weights_of=3)])))      # through a layer that borrows itself
    m5 = sutosun.Config.from_json(chain)
    assert [m5.source(i) for i in range(5)] == [0, 1, 2, 1, 1] and m5.tensor_shapes() == m.tensor_shapes()
    chain["layers"][3]["weights_of"] = 4
    with pytest.raises(ValueError):
        sutosun.Config.from_json(chain)
    plain = json.loads(json.dumps(cfg))           # what a configuration leaves out does not exist
    del plain["logit_softcap"], plain["layers"][0]["mixer"]["rot"]
    for l in (1, 3):
        del plain["layers"][l]["mixer"]["q_temp"]
    assert sutosun.Config.from_json(plain).logit_softcap == 0.0


def test_checkpoint_names_and_shapes_match_the_reference_listing():
    from atx.models import sutosun

    cfg = small_cfg()
    names = R.checkpoint_shapes(cfg)
    assert sutosun.Config.from_json(cfg).tensor_shapes() == names
    assert names["embed.norm"] == (48,) and names["head"] == (90, 48) and "l2.norm2" not in names
    assert not any(k.startswith("l3.") for k in names)
    assert names["l1.mix.q.norm"] == (72,) and names["l1.mix.k.b"] == (24,) and names["l1.mix.v"] == (20, 48) and names["l1.mix.g"] == (6, 48)
    assert names["l2.mix.q"] == (40, 48) and names["l2.mix.dkv"] == (24, 48) and names["l2.mix.sink"] == (4,)
    assert names["l0.mlp.router.b"] == (5,) and names["l0.mix.g"] == (42, 48) and "l0.mix.norm" not in names


def test_weights_are_stacked_the_way_the_kernels_read_them():
    from atx.models import sutosun

    cfg = small_cfg()
    wt = R.random_checkpoint(cfg, 1)
    m = sutosun.Config.from_json(cfg)
    w = sutosun.Weights.from_state_dict(m, wt, torch.device("cpu"), torch.float32)
    l0, l1, l2, l3 = w.layers
    assert l3 is l1
    assert l1.w_in.shape == (72 + 24 + 20 + 6, 48) and torch.equal(l1.w_in[96:116].double(), wt["l1.mix.v"])
    assert torch.equal(l1.bk.double(), wt["l1.mix.k.b"]) and l1.sinks.dtype == torch.float32
    assert l0.w_in.shape == (24 + 24 + 42 + 42, 48) and l0.decay.tolist() == torch.tensor([0.5, 0.9, 0.99]).tolist()
    assert l2.w_ukt.shape == (4 * 20, 6) and torch.equal(l2.w_ukt[20:40].double(), wt["l2.mix.uk"][6:12].T) and l2.norm2 is None
    assert l0.w_gu.shape == (5, 48, 48) and torch.equal(l0.w_gu[3, 24:].double(), wt["l0.mlp.e3.up"]) and not l0.gu_interleaved
    assert l1.w_gu.shape == (80, 48) and torch.equal(l0.router_b.double(), wt["l0.mlp.router.b"])
    n = sum(t.numel() for t in wt.values())
    assert w.nbytes() == 4 * (n + 3)               # every tensor once, and the three decays
    sd = dict(wt)
    del sd["l0.mlp.router.b"]
    with pytest.raises(KeyError):
        sutosun.Weights.from_state_dict(m, sd, torch.device("cpu"), torch.float32)
    with pytest.raises(ValueError):
        sutosun.Weights.from_state_dict(m, dict(wt, **{"l1.mix.q.norm": torch.zeros(12)}), torch.device("cpu"), torch.float32)


def test_gate_and_up_rows_are_interleaved_where_the_gated_gemm_reads_them():
    from atx.models.common import gate_up_matrix

    g, u = torch.arange(128.0)[:, None].expand(128, 64), 1000.0 + torch.arange(128.0)[:, None].expand(128, 64)
    m, inter = gate_up_matrix(g, u, 64, torch.bfloat16)
    assert inter and m.shape == (256, 64)
    assert m[:, 0].tolist() == g[:64, 0].tolist() + u[:64, 0].tolist() + g[64:, 0].tolist() + u[64:, 0].tolist()
    for args in ((g, u, 64, torch.float32), (g, u, 72, torch.bfloat16), (g[:100], u[:100], 64, torch.bfloat16)):
        m, inter = gate_up_matrix(*args)
        assert not inter and torch.equal(m, torch.cat(args[:2], 0))


def test_named_shapes_come_through_the_registry():
    from atx.config import resolve_model

    for name, layers in (("sutosun-tiny", 4), ("sutosun-1b", 16), ("sutosun-8b", 32)):
        c = resolve_model(f"random:{name}:1").config
        assert c.architecture == "Sutosun" and c.num_hidden_layers == layers
        assert [l["type"] for l in c.layers[:4]] == ["retention", "latent_attention", "attention", "retention"]
        assert all(0.9 < d < 1.0 for d in c.layers[0]["mixer"]["decay"])
    assert c.weight_bytes_per_decode_step(2, 8) > c.weight_bytes_per_decode_step(2, 1)     # more tokens reach more experts
    shared = json.loads(json.dumps(c.layers))
    shared[4] = dict(shared[0], weights_of=0)
    s = type(c)(**dict(vars(c), layers=shared))
    assert s.weight_bytes_per_decode_step(2, 8) == c.weight_bytes_per_decode_step(2, 8)    # streamed again where they are used again


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
    sch.retire(a)
    plan = sch.plan_explicit([(b, 2, [1])])
    assert len(plan.prefills) == 1 and b.state_slot == 0 and slots.num_free == 0 and alloc.num_free == 7


def test_reference_recurrence_equals_its_sum_over_pairs():
    g = torch.Generator().manual_seed(0)
    q, k, v = torch.randn(23, 6, generator=g, dtype=F64), torch.randn(23, 6, generator=g, dtype=F64), torch.randn(23, 5, generator=g, dtype=F64)
    for decay in (1.0, 0.97, 0.3, 0.0):
        a, b = R.decayed_outer_recurrence(q, k, v, decay), R.decayed_pair_sum(q, k, v, decay)
        assert torch.allclose(a, b), decay
    assert torch.allclose(R.decayed_outer_recurrence(q, k, v, 0.0), (q * k).sum(-1, keepdim=True) * v)


def test_reference_sink_factor_rotation_and_routing():
    g = torch.Generator().manual_seed(1)
    # one key: weight e^s / (e^s + e^sink), the sink not scaled
    q = torch.tensor([[[2.0, 0.0]], [[2.0, 0.0]]], dtype=F64)
    k = torch.tensor([[[1.0, 0.0]], [[-50.0, 0.0]]], dtype=F64)
    v = torch.tensor([[[3.0, 1.0]], [[7.0, 7.0]]], dtype=F64)
    o = R.sink_attention(q, k, v, 0.5, torch.tensor([0.25], dtype=F64))
    w = math.exp(1.0) / (math.exp(1.0) + math.exp(0.25))
    assert torch.allclose(o[0, 0], w * v[0, 0]) and torch.allclose(o[1, 0], w * v[0, 0])
    assert float(R.sink_attention(q, k, v, 0.5, torch.tensor([80.0], dtype=F64)).abs().max()) < 1e-30
    # heads in groups: head h reads key/value head h // (H / G)
    q, k, v = (torch.randn(5, n, 4, generator=g, dtype=F64) for n in (6, 2, 2))
    sk = torch.randn(6, generator=g, dtype=F64)
    o = R.sink_attention(q, k, v, 0.7, sk)
    assert torch.allclose(o[:, 4:5], R.sink_attention(q[:, 4:5], k[:, 1:], v[:, 1:], 0.7, sk[4:5]))
    # the factor is 1 up to position every - 2 and grows by steps at every-th positions
    f = R.query_factor(12, 0.5, 4)
    assert f[:3].tolist() == [1.0] * 3 and torch.allclose(f[3:7], torch.full((4,), 1 + 0.5 * math.log(2.0), dtype=F64))
    assert abs(float(f[11]) - (1 + 0.5 * math.log(4.0))) < 1e-12
    # rotation pairs element i with i + half, keeps lengths, leaves position 0 and the rest
    x = torch.randn(5, 2, 8, generator=g, dtype=F64)
    fr, mag = R.pair_frequencies(6, 50.0)
    y = R.rotate_halves(x, fr, mag)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    assert torch.allclose(y[..., :3] ** 2 + y[..., 3:6] ** 2, x[..., :3] ** 2 + x[..., 3:6] ** 2)
    assert torch.allclose(y[3, 0, 0], x[3, 0, 0] * math.cos(3.0) - x[3, 0, 3] * math.sin(3.0))
    # stretched frequencies: the fast pairs stay, the slow ones are divided, the magnitude is on cos and sin
    sc = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    fs, mag = R.pair_frequencies(64, 10000.0, sc)
    f0, _ = R.pair_frequencies(64, 10000.0)
    assert float(fs[0]) == float(f0[0]) and abs(float(fs[-1] / f0[-1]) - 1 / 8) < 1e-12 and abs(mag - (0.1 * math.log(8.0) + 1)) < 1e-12
    # routing: the bias moves the choice and the weights; the weights are a soft-max over the chosen outputs alone
    h, router = torch.randn(6, 4, generator=g, dtype=F64), torch.randn(5, 4, generator=g, dtype=F64)
    bias = torch.tensor([0.0, 0.0, 30.0, 0.0, 0.0], dtype=F64)
    idx, wgt = R.route(h, router, bias, 2)
    z = h @ router.T + bias
    assert bool((idx[:, 0] == 2).all()) and torch.allclose(wgt, torch.softmax(z.gather(1, idx), -1)) and torch.allclose(wgt.sum(-1), torch.ones(6, dtype=F64))
    full = torch.softmax(z, -1).gather(1, idx)
    assert torch.allclose(wgt, full / full.sum(-1, keepdim=True))       # which is how the kernel forms them
    z = torch.linspace(-6, 6, 101, dtype=F64)
    assert torch.allclose(R.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh")) and torch.allclose(R.silu(z), z * torch.sigmoid(z))
    assert torch.allclose(R.gelu_tanh(z), z * torch.sigmoid(2 * math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def test_product_frequencies_match_the_reference():
    from atx.models.common import stretched_frequencies

    for dims, base, sc in ((6, 100.0, None), (4, 50.0, {"factor": 3.0, "original": 40, "fast": 4.0, "slow": 0.5}),
                           (64, 500000.0, {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}),
                           (8, 4.0, {"factor": 8.0, "original": 64, "fast": 64.0, "slow": 0.01}), (2, 10.0, {"factor": 2.0, "original": 9, "fast": 2.0, "slow": 2.0})):
        f, mag = stretched_frequencies(base, dims, sc)
        want, wmag = R.pair_frequencies(dims, base, sc)
        assert torch.allclose(torch.tensor(f, dtype=F64), want) and mag == wmag


def test_reference_is_causal_and_a_layer_may_run_another_layers_tensors():
    cfg = small_cfg()
    wt = R.random_checkpoint(cfg, 2)
    toks = [int(t) for t in torch.randint(0, 90, (19,), generator=torch.Generator().manual_seed(0))]
    a = R.forward(cfg, wt, toks)
    assert torch.allclose(a[:12], R.forward(cfg, wt, toks[:12])) and a.shape == (19, 90) and float(a.abs().max()) < 12.0
    own = json.loads(json.dumps(cfg))
    del own["layers"][3]["weights_of"]
    copied = dict(wt, **{k.replace("l1.", "l3.", 1): t for k, t in wt.items() if k.startswith("l1.")})
    assert torch.equal(R.forward(own, copied, toks), a)
    # silent layers leave the normed embedding
    quiet = {k: (torch.zeros_like(t) if k.endswith("mix.o") or k.endswith(".down") else t) for k, t in wt.items()}
    res = []
    R.forward(cfg, quiet, toks, res)
    e = wt["embed"][toks]
    want = e / torch.sqrt((e * e).mean(-1, keepdim=True) + 1e-5) * wt["embed.norm"]
    assert all(torch.allclose(x, want) for x in res)

"""Host-side checks of the Korirax design (no GPU): configuration reader and registry, tensor names and shapes, synthetic weights,
and the oracle's mechanisms against closed forms written out in the tests themselves."""
import json
import math

import pytest
import torch

from moshi_b200.config import DECODER_ARCHITECTURES, DecoderLMConfig, KoriraxConfig
from moshi_b200.synth import iter_synth_decoder_tensors
from oracle import korirax as K

F64 = torch.float64


def small_cfg():
    return {"architecture": "Korirax", "embedding": {"scale": 1.5}, "norm": {"eps": 1e-5}, "vocab": 31, "width": 12, "token_side": {"dim": 3},
            "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": [{"type": "rglru", "mixer": {"blocks": 3, "conv": 4, "width": 6}, "mlp": {"ff": 9, "kind": "dense"}},
                       {"type": "latent_attention", "mixer": {"dim": 5, "heads": 2, "kv_rank": 7, "q_rank": 9, "rot_dim": 4, "scale": 0.3, "vdim": 6,
                                                              "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0, "fast": 8.0, "original": 64, "slow": 1.0}}},
                        "mlp": {"expert": {"ff": 7}, "kind": "moe", "router": {"experts": 6, "groups": {"count": 3, "keep": 2}, "scale": 1.7, "top": 3}, "shared": {"ff": 11}}},
                       {"type": "attention", "mixer": {"bias_max": 20.0, "dim": 4, "heads": 4, "kv_heads": 2, "q_temp": {"coef": 0.2, "every": 5.0}, "scale": 0.4, "vdim": 3},
                        "mlp": None},
                       {"type": "attention", "mixer": {"bias_max": 40.0, "dim": 4, "heads": 2, "kv_heads": 1, "scale": 0.4, "vdim": 3},
                        "mlp": {"expert": {"ff": 8}, "kind": "moe", "router": {"experts": 3, "scale": 1.0, "top": 1}}}]}


def test_configuration_round_trip_and_registry():
    raw = small_cfg()
    cfg = DecoderLMConfig.from_dict(raw)
    assert isinstance(cfg, KoriraxConfig) and DECODER_ARCHITECTURES["Korirax"] is KoriraxConfig
    assert cfg.block == "parallel_residual" and cfg.norm == "rms" and cfg.embedding_scale == 1.5 and cfg.side_dim == 3 and not cfg.tied_head
    a, b, c, d = cfg.layers
    assert a.a.kind == "rglru" and a.a.dim == 6 and a.a.blocks == 3 and a.a.conv == 4 and a.mlp_kind == "silu_glu"
    assert b.a.q_rank == 9 and b.a.rot_dims == 4 and b.a.rot_pairing == "adjacent" and b.a.rot_scaling_kind == "ramp" and b.a.out_gate and b.a.sink == "none"
    assert b.mlp_kind == "moe_gelu" and b.experts == 6 and b.top == 3 and b.groups == 3 and b.groups_keep == 2 and b.router_scale == 1.7 and b.shared_ff == 11
    assert c.a.kind == "bias_attention" and c.a.bias_max == 20.0 and c.a.q_temp_coef == 0.2 and c.a.q_temp_every == 5.0 and c.a.qk_norm and c.a.bias and c.mlp_kind is None
    assert d.a.q_temp_every == 0.0 and d.groups == 1 and d.shared_ff == 0
    assert cfg.layer_runs() == [0, 1, 2, 1, 2, 3] and [i for i, _ in K.layer_runs(raw)] == cfg.layer_runs()
    assert [t for _, t in K.layer_runs(raw)] == [None, 0, None, 1, None, None]
    assert json.loads(json.dumps(cfg.to_dict())) == raw
    plain = small_cfg()
    del plain["loop"], plain["token_side"]
    c2 = DecoderLMConfig.from_dict(plain)
    assert c2.to_dict() == plain and c2.layer_runs() == [0, 1, 2, 3] and not any("side" in k or "loop" in k for k in c2.tensor_shapes())
    from moshi_b200.models.loaders import model_class
    assert model_class(raw).__name__ == "DecoderLM"
    for edit in (lambda x: x["layers"][0].update(type="delta"), lambda x: x["layers"][0]["mlp"].update(kind="other"), lambda x: x["loop"].update(stop=5),
                 lambda x: x["loop"].update(times=0), lambda x: x["layers"][0]["mixer"].update(blocks=4), lambda x: x["layers"][1]["mixer"]["rot"].update(dims=2)):
        bad = small_cfg()
        edit(bad)
        with pytest.raises(ValueError):
            DecoderLMConfig.from_dict(bad)


def test_tensor_names_and_synthetic_weights():
    cfg = DecoderLMConfig.from_dict(small_cfg())
    s = cfg.tensor_shapes()
    assert s["loop.step"] == (2, 12) and s["side.embed"] == (31, 12) and s["l3.side.gate"] == (3, 12) and s["l3.side.proj"] == (12, 3) and s["l0.side.norm"] == (12,)
    assert s["l0.mix.y"] == (6, 12) and s["l0.mix.x.b"] == (6,) and s["l0.mix.conv"] == (6, 4) and s["l0.mix.ra"] == (3, 2, 2) and s["l0.mix.ri.b"] == (3, 2) and s["l0.mix.o"] == (12, 6)
    assert s["l1.mix.dq"] == (9, 12) and s["l1.mix.uq"] == (18, 9) and s["l1.mix.dkv"] == (11, 12) and s["l1.mix.uk"] == (10, 7) and s["l1.mix.g"] == (12, 12)
    assert s["l1.mlp.e5.up"] == (7, 12) and "l1.mlp.e5.gate" not in s and s["l1.mlp.shared.down"] == (12, 11) and s["l1.mlp.router"] == (6, 12)
    assert s["l2.mix.q"] == (16, 12) and s["l2.mix.k.b"] == (8,) and s["l2.mix.rel"] == (32, 4) and s["l2.mix.k.norm"] == (4,) and "l2.mlp.router" not in s
    t = dict(iter_synth_decoder_tensors(cfg, seed=1))
    assert set(t) == set(s) and all(tuple(t[k].shape) == s[k] for k in s)
    assert float(t["l0.norm1"].float().min()) > 0.5 and float(t["l0.mix.lam"].float().max()) < -2.0
    lg, layers = K.Oracle(cfg.to_dict(), t).run([3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5])
    assert lg.shape == (11, 31) and layers.shape == (6, 11, 12) and bool(torch.isfinite(lg).all())


def test_distance_buckets():
    b = [K.distance_bucket(n, 8, 64) for n in range(200)]
    # four rows of their own, then a row per factor 2 (ln(n / 4) / ln(16) * 4 = log2(n / 4))
    assert b[:4] == [0, 1, 2, 3] and b[4:8] == [4] * 4 and b[8:16] == [5] * 8 and set(b[32:]) == {7}
    assert all(x <= y for x, y in zip(b, b[1:])) and K.distance_bucket(10 ** 6, 8, 64) == 7
    odd = [K.distance_bucket(n, 20, 70) for n in range(100)]
    assert odd[9] == 9 and odd[10] == 10 and odd[12] == 10 and odd[13] == 11 and odd[57] == 18 and odd[58] == 19 and odd[99] == 19


def test_query_temperature_steps():
    assert K.temperature(0, 0.5, 4) == 1.0 and K.temperature(2, 0.5, 4) == 1.0
    assert abs(K.temperature(3, 0.5, 4) - (1 + 0.5 * math.log(2))) < 1e-15 and K.temperature(6, 0.5, 4) == K.temperature(3, 0.5, 4)
    assert abs(K.temperature(11, 0.3, 4) - (1 + 0.3 * math.log(4))) < 1e-15


def test_rotation_ramp_by_hand():
    f, amp = K.rotary(8, 100.0)
    assert amp == 1.0 and torch.allclose(f, torch.tensor([100.0 ** (-i / 4) for i in range(4)], dtype=F64))
    sc = {"factor": 4.0, "original": 200.0, "fast": 8.0, "slow": 1.0}
    g, amp = K.rotary(8, 100.0, sc)
    index = [8 * math.log(200.0 / (2 * math.pi * t)) / (2 * math.log(100.0)) for t in (8.0, 1.0)]      # 1.20 and 3.01
    lo, hi = math.floor(index[0]), math.ceil(index[1])
    assert (lo, hi) == (1, 4) and abs(amp - (0.1 * math.log(4.0) + 1)) < 1e-15
    want = [float(f[i]) * (1 - r) + float(f[i]) / 4 * r for i, r in enumerate((0.0, 0.0, 1 / 3, 2 / 3))]
    assert torch.allclose(g, torch.tensor(want, dtype=F64), atol=1e-15)
    e = torch.zeros(2, 8, dtype=F64)
    e[1, 2] = 1.0
    r = K.rotate_adjacent(e, 3, f, 2.0)
    assert abs(float(r[1, 2]) - 2 * math.cos(3 * float(f[1]))) < 1e-14 and abs(float(r[1, 3]) - 2 * math.sin(3 * float(f[1]))) < 1e-14


def test_attention_of_one_head_by_hand():
    g = torch.Generator().manual_seed(3)
    W, d, dv = 5, 3, 2
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    p = {"q": r(d, W), "q.b": r(d), "k": r(d, W), "k.b": r(d), "v": r(dv, W), "v.b": r(dv), "q.norm": r(d), "k.norm": r(d), "rel": r(4, 1), "g": r(dv, W), "o": torch.eye(dv, dtype=F64)}
    m = {"heads": 1, "kv_heads": 1, "dim": d, "vdim": dv, "scale": 0.8, "bias_max": 3, "q_temp": {"coef": 0.4, "every": 2}}
    hs, st = r(4, W), {}
    for t in range(4):
        out = K.attention(p, m, hs[t], t, st, 1e-5)
    unit = lambda u: u / torch.sqrt((u * u).mean() + 1e-5)
    q = unit(p["q"] @ hs[3] + p["q.b"]) * p["q.norm"] * (1 + 0.4 * math.log(3))
    rows = {0: 0, 1: 1, 2: 2, 3: 3}                       # distance 2: 2 + floor(0), distance 3: the last row
    s = torch.stack([(unit(p["k"] @ hs[j] + p["k.b"]) * p["k.norm"]) @ q * 0.8 + p["rel"][rows[3 - j], 0] for j in range(4)])
    w = torch.softmax(s, 0)
    want = sum(w[j] * (p["v"] @ hs[j] + p["v.b"]) for j in range(4)) * torch.sigmoid(p["g"] @ hs[3])
    assert torch.allclose(out, want, atol=1e-12)


def test_latent_attention_by_hand():
    g = torch.Generator().manual_seed(4)
    W, d, rd, dv, r, qr = 6, 3, 2, 2, 4, 5
    rn = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    p = {"dq": rn(qr, W), "dq.norm": rn(qr), "uq": rn(d + rd, qr), "dkv": rn(r + rd, W), "dkv.norm": rn(r), "uk": rn(d, r), "uv": rn(dv, r), "g": rn(dv, W), "o": torch.eye(dv, dtype=F64)}
    m = {"heads": 1, "dim": d, "rot_dim": rd, "vdim": dv, "kv_rank": r, "q_rank": qr, "scale": 0.6, "rot": {"base": 50.0, "dims": rd}}
    hs, st = rn(2, W), {}
    for t in range(2):
        out = K.latent_attention(p, m, hs[t], t, st, 1e-5)
    unit = lambda u: u / torch.sqrt((u * u).mean() + 1e-5)
    turn = lambda u, a: torch.stack([u[0] * math.cos(a) - u[1] * math.sin(a), u[1] * math.cos(a) + u[0] * math.sin(a)])
    q = p["uq"] @ (unit(p["dq"] @ hs[1]) * p["dq.norm"])
    c = [unit((p["dkv"] @ h)[:r]) * p["dkv.norm"] for h in hs]
    s = torch.stack([((p["uk"] @ c[j]) @ q[:d] + turn((p["dkv"] @ hs[j])[r:], float(j)) @ turn(q[d:], 1.0)) * 0.6 for j in range(2)])
    w = torch.softmax(s, 0)
    assert torch.allclose(out, (w[0] * (p["uv"] @ c[0]) + w[1] * (p["uv"] @ c[1])) * torch.sigmoid(p["g"] @ hs[1]), atol=1e-12)


def test_recurrence_unrolled_and_convolution_as_a_sum():
    g = torch.Generator().manual_seed(5)
    W, n, taps = 4, 6, 3
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    p = {"y": r(n, W), "y.b": r(n), "x": r(n, W), "x.b": r(n), "conv": r(n, taps), "conv.b": r(n), "ra": r(2, 3, 3), "ra.b": r(2, 3), "ri": r(2, 3, 3), "ri.b": r(2, 3),
         "lam": r(n) - 2.0, "o": torch.eye(n, dtype=F64)}
    hs, st = r(5, W), {}
    outs = [K.rglru(p, {}, hs[t], t, st, 1e-5) for t in range(5)]
    x = [p["x"] @ h + p["x.b"] for h in hs]
    S = torch.zeros(n, dtype=F64)
    for t in range(5):
        u = p["conv.b"] + sum(p["conv"][:, taps - 1 - k] * x[t - k] for k in range(taps) if t - k >= 0)
        gate = lambda nm: torch.sigmoid(torch.cat([p[nm][b] @ u[3 * b:3 * b + 3] for b in range(2)]) + p[nm + ".b"].reshape(-1))
        a = torch.exp(-8.0 * gate("ra") * torch.nn.functional.softplus(p["lam"]))
        S = a * S + torch.sqrt(1 - a * a) * gate("ri") * u
        y = torch.nn.functional.gelu(p["y"] @ hs[t] + p["y.b"], approximate="tanh")
        assert torch.allclose(outs[t], S * y, atol=1e-10)


def test_router_groups_by_their_two_best_and_renormalised_weights():
    s = torch.tensor([0.60, 0.10, 0.50, 0.45, 0.20, 0.30], dtype=F64)
    z = torch.log(s / (1 - s))
    none = torch.zeros(6, dtype=F64)
    idx, w = K.route(z, none, 2, 1, 1, 2.0)
    assert idx == [0, 2] and abs(w[0] - 0.6 / 1.1 * 2) < 1e-12 and abs(w[1] - 0.5 / 1.1 * 2) < 1e-12
    idx, _ = K.route(z, none, 2, 3, 1, 1.0)
    assert idx == [2, 3]                                                                   # 0.95 against 0.70: not the group with the largest single score
    corr = none.clone()
    corr[1] = 0.5
    idx, w = K.route(z, corr, 1, 3, 1, 1.0)
    assert idx == [0] and abs(w[0] - 1.0) < 1e-12                                          # 1.20: the correction moves the group, the weight is the plain score
    idx, _ = K.route(z, none - 5.0, 2, 3, 1, 1.0)                                          # negative choice scores: the other groups stay out
    assert idx == [2, 3]
    g = torch.Generator().manual_seed(6)
    W, F = 4, 3
    p = {"router": torch.zeros(2, W, dtype=F64), "correction": torch.tensor([0.0, 1.0], dtype=F64)}
    for e in ("e0", "e1", "shared"):
        p.update({f"{e}.up": torch.randn(F, W, generator=g, dtype=F64), f"{e}.down": torch.randn(W, F, generator=g, dtype=F64)})
    h = torch.randn(W, generator=g, dtype=F64)
    want = sum(c * p[f"{e}.down"] @ torch.nn.functional.gelu(p[f"{e}.up"] @ h) for e, c in (("e1", 2.5), ("shared", 1.0)))
    assert torch.allclose(K.experts(p, {"router": {"experts": 2, "top": 1, "scale": 2.5}, "shared": {"ff": F}}, h), want, atol=1e-12)


def test_token_input_and_silu_unit_by_hand():
    eye = torch.eye(2, dtype=F64)
    x, e = torch.tensor([0.5, -1.0], dtype=F64), torch.tensor([2.0, 3.0], dtype=F64)
    y = torch.nn.functional.gelu(x, approximate="tanh") * e
    got = K.token_input({"gate": eye, "proj": eye, "norm": torch.tensor([1.0, 0.5], dtype=F64)}, x, e, 1e-3)
    assert torch.allclose(got, y / math.sqrt(float((y * y).mean()) + 1e-3) * torch.tensor([1.0, 0.5], dtype=F64), atol=1e-12)
    assert torch.allclose(K.silu_glu({"gate": eye, "up": 2 * eye, "down": eye}, x), torch.nn.functional.silu(x) * 2 * x, atol=1e-14)


def test_state_is_carried_over_a_cut_and_owned_by_every_pass():
    cfg = DecoderLMConfig.from_dict(small_cfg())
    t = dict(iter_synth_decoder_tensors(cfg, seed=2))
    o = K.Oracle(cfg.to_dict(), t)
    toks = [3, 7, 7, 1, 0, 30, 12, 5, 9, 2, 2, 8]
    whole, _ = o.run(toks)
    st = o.new_state()
    a, _ = o.run(toks[:4], st)
    b, _ = o.run(toks[4:], st)
    assert torch.equal(torch.cat([a, b]), whole)
    assert len(st["runs"]) == 6 and st["runs"][1]["c"] is not st["runs"][3]["c"] and not torch.equal(st["runs"][1]["c"][3], st["runs"][3]["c"][3])
    assert st["runs"][0]["S"].shape == (6,) and len(st["runs"][0]["u"]) == 4

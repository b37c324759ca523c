"""Dedunex without a GPU: the configuration's reader and its errors, the model as data (parts, tensors, run order, cache
and state needs), the scaled rotation's frequencies, and the plain implementation's own checks against formulas written
out element by element."""
import json
import math

import pytest
import torch

from dedunex_util import config, dense, diff_layer, gru_layer, latent_layer, write_model


def build(cfg_dict):
    from nanoinfer_b200.config import DedunexConfig
    from nanoinfer_b200.models.model import Model
    from nanoinfer_b200.registry import get_architecture

    cfg = DedunexConfig.from_dict(json.loads(json.dumps(cfg_dict)))
    return Model(get_architecture(cfg.architecture).build_spec(cfg), cfg)


def test_the_architecture_is_registered():
    from nanoinfer_b200 import architectures
    from nanoinfer_b200.config.base import architecture_name

    assert {"Dedunex", "Nagilix", "Kemuzen", "Mulavik", "Vadonex", "GPT2LMHeadModel"} <= set(architectures())
    assert architecture_name({"architecture": "Dedunex"}) == "Dedunex"


def test_all_problems_of_a_configuration_come_in_one_error():
    from nanoinfer_b200.config import ConfigError, DedunexConfig

    bad = config([diff_layer(heads=3, kv_heads=2), latent_layer(), dict(type="conv", mixer={}), gru_layer(mlp=dict(kind="moe")),
                  diff_layer(dim=8, rot=10), diff_layer(), latent_layer(), diff_layer(dim=200)], width=64, groups=3,
                 loop=(2, 9, 0))
    del bad["layers"][1]["mixer"]["q_rank"]
    del bad["layers"][5]["mixer"]["rot"]["scaling"]["slow"]
    bad["layers"][6]["mixer"]["rot"]["scaling"] = dict(factor=2.0, original=10, fast=1.0, slow=1.0)
    bad["norm"].pop("eps")
    with pytest.raises(ConfigError) as e:
        DedunexConfig.from_dict(bad)
    text = str(e.value)
    for piece in ("norm.eps", "norm.groups", "loop: start 2 and stop 9", "loop.times", "layers[0].mixer.heads",
                  "layers[1].mixer.q_rank", "layers[2].type", "layers[3].mlp.kind", "layers[4].mixer.rot.dims",
                  "layers[5].mixer.rot.scaling.slow", "layers[6].mixer.rot.scaling", "layers[7].mixer.dim"):
        assert piece in text, (piece, text)


def test_defaults_of_keys_that_may_be_left_out():
    cfg = config([diff_layer(softcap=0, window=0, rot=0), latent_layer(rot_dim=0)])
    del cfg["layers"][0]["mixer"]["kv_heads"], cfg["norm"]["groups"]
    m = build(cfg)
    a, lat = m.layers[0].mixer, m.layers[1].mixer
    assert a.n_kv_head == a.n_head and a.window == 0 and a.softcap == 0.0 and a.position is None
    assert lat.rot_dims == 0 and lat.halves and lat.head_gate
    assert m.layers[0].norm_1.groups == 1 and m.stream_vectors is None and m.layers[0].feed_forward is None
    assert [e.add_vector for e in m.schedule] == [None, None]


def test_run_order_parts_tensors_cache_and_state_of_a_looped_stack():
    from nanoinfer_b200.cache import CacheManager

    layers = [gru_layer(width=24), diff_layer(heads=4, kv_heads=2, dim=16, vdim=40, window=24, mlp=dense(32)),
              latent_layer(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=20, kv_rank=32), gru_layer(width=40, mlp=dense(16)),
              diff_layer(heads=2, kv_heads=1, dim=40, vdim=24, window=0)]
    m = build(config(layers, vocab=99, width=64, groups=4, loop=(1, 4, 3)))
    assert [(e.layer, e.add_vector) for e in m.schedule] == [(0, None), (1, 0), (2, None), (3, None), (1, 1), (2, None),
                                                             (3, None), (1, 2), (2, None), (3, None), (4, None)]
    assert [type(b).__name__ for b in m.layers] == ["ParallelNormBlock"] * 5
    assert [b.joint for b in m.layers] == [False, True, False, True, False]
    names = {b.ref.name: tuple(b.spec.shape) for b in m.bindings()}
    assert names["embed.norm"] == (64,) and names["loop.step"] == (3, 64) and names["final.norm"] == (64,)
    assert names["l1.mix.q"] == (128, 64) and names["l1.mix.k"] == (64, 64) and names["l1.mix.v.b"] == (80,)
    assert names["l1.mix.q.norm"] == (16,) and names["l1.mix.lk2"] == (16,) and names["l1.mix.o"] == (64, 160)
    assert names["l2.mix.dkv"] == (40, 64) and names["l2.mix.uq"] == (72, 20) and names["l2.mix.g"] == (3, 64)
    assert names["l3.mix.x.b"] == (40,) and names["l3.mlp.down"] == (64, 16) and "l0.mlp.gate" not in names
    # every run of a looped layer has pages, or a state, of its own
    kv = dict(m.kv_needs())
    assert set(kv) == {1, 2, 4, 5, 7, 8, 10}
    assert (kv[4].n_kv_head, kv[4].head_dim, kv[4].window, kv[4].planes) == (2, 48, 24, 2)       # max(2 * 16, 40) -> 48
    assert (kv[5].n_kv_head, kv[5].head_dim, kv[5].planes) == (1, 40, 1) and kv[10].head_dim == 80
    st = dict(m.state_needs())
    assert set(st) == {0, 3, 6, 9} and st[0].shape == (24,) and st[9].shape == (40,)
    cm = CacheManager(m.kv_needs(), m.state_needs(), max_tokens=128, max_requests=2, page_size=16)
    assert len(cm.groups) == 3


def test_a_loop_of_one_pass_still_adds_its_vector():
    m = build(config([gru_layer(), gru_layer()], loop=(1, 2, 1)))
    assert [(e.layer, e.add_vector) for e in m.schedule] == [(0, None), (1, 0)] and m.stream_vectors.count == 1


@pytest.mark.parametrize("base,dims,sc", [(10000.0, 16, dict(factor=4.0, original=1024, fast=32.0, slow=1.0)),
                                          (500.0, 12, dict(factor=2.5, original=64, fast=4.0, slow=0.5)),
                                          (1e6, 64, dict(factor=16.0, original=4096, fast=32.0, slow=1.0)),
                                          (50.0, 4, dict(factor=8.0, original=7, fast=1.0, slow=1.0)),
                                          (100.0, 2, dict(factor=1.0, original=50, fast=2.0, slow=1.0))])
def test_scaled_rotation_frequencies(base, dims, sc):
    """Against the rule written out with one loop and if-clauses: wavelengths much shorter than the original length stay,
    much longer ones are stretched by the factor."""
    from nanoinfer_b200.parts.base import POSITIONS

    part = POSITIONS.build("rotary_halves", base=base, dims=dims, scaling=sc)
    idx = lambda t: dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = math.floor(idx(sc["fast"])), math.ceil(idx(sc["slow"]))
    lo, hi = (0 if lo < 0 else lo), (dims - 1 if hi > dims - 1 else hi)
    span = hi - lo if hi - lo > 0.001 else 0.001
    for i, got in enumerate(part.frequencies()):
        plain = base ** (-2.0 * i / dims)
        if i <= lo:
            want = plain if i < lo or (i - lo) / span <= 0 else None
        elif (i - lo) / span >= 1:
            want = plain / sc["factor"]
        else:
            r = (i - lo) / span
            want = plain * (1 - r) + plain * r / sc["factor"]
        assert want is None or abs(got - want) < 1e-15 * max(1.0, plain) + 1e-12 * want, i
    assert part.amplitude == 0.1 * math.log(sc["factor"]) + 1.0
    plain = POSITIONS.build("rotary_halves", base=base, dims=dims)
    assert plain.amplitude == 1.0 and plain.frequencies() == [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    import plain_dedunex as P
    f, amp = P.rotary_frequencies(dict(base=base, dims=dims, scaling=sc))
    assert torch.allclose(f, torch.tensor(part.frequencies(), dtype=torch.float64), rtol=1e-13, atol=0) and amp == part.amplitude


def test_random_weights_fit_the_model_and_the_plain_model_reads_them(tmp_path):
    from plain_dedunex import PlainDedunex

    cfg = config([diff_layer(mlp=dense()), latent_layer(mlp=dense()), gru_layer()], vocab=70, width=32, loop=(0, 2, 2))
    d = write_model(cfg, str(tmp_path), torch.float32, seed=2)
    layers = []
    out = PlainDedunex(d).logits(list(range(30)), layers)
    assert out.shape == (30, 70) and bool(torch.isfinite(out).all()) and float(out.std()) > 0.1 and len(layers) == 5


def test_joint_products_keep_every_parameter_in_its_place():
    """A layer whose two sublayers share their products: the parameters by name are views of the joint matrices and hold
    what was loaded."""
    m = build(config([diff_layer(heads=2, kv_heads=1, dim=10, vdim=14, mlp=dense(12)), latent_layer(mlp=dense(20)),
                      gru_layer(width=13, mlp=dense(9))], width=32))
    g = torch.Generator().manual_seed(0)
    want = {}
    per = {}
    for b in m.bindings():
        t = torch.randn(b.spec.shape, generator=g)
        want[(id(b.part), b.spec.key)] = t
        per.setdefault(id(b.part), (b.part, {}))[1][b.spec.key] = t.clone()
    for part, params in per.values():
        part.bind(params)
    for part in m.all_parts():
        if not hasattr(part, "params"):
            part.bind({})
    m.prepare(torch.float32, torch.device("cpu"))
    for b in m.bindings():
        assert torch.equal(b.part.params[b.spec.key], want[(id(b.part), b.spec.key)]), (b.where, b.spec.key)
    for blk in m.layers:
        for part in (blk.mixer, blk.feed_forward):
            assert part.w_in.untyped_storage().data_ptr() == blk.w_in.untyped_storage().data_ptr()
            assert part.w_out.untyped_storage().data_ptr() == blk.w_out.untyped_storage().data_ptr()
        x = torch.randn(5, 32, generator=g)
        whole = x @ blk.w_in.T
        assert torch.allclose(whole[:, :blk.mixer.n_in], x @ blk.mixer.w_in.T)
        assert torch.allclose(whole[:, blk.ff_row:blk.ff_row + blk.feed_forward.n_in], x @ blk.feed_forward.w_in.T)


# --------------------------------------------------------------------------- the plain model against written-out formulas
def test_plain_differential_attention_element_by_element():
    import plain_dedunex as P

    torch.manual_seed(0)
    n, C, H, G, d, dv, size, eps = 9, 10, 4, 2, 4, 3, 4, 1e-5
    m = dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=0.7, softcap=1.5, diff=0.3, mask=dict(size=size), rot=dict(dims=2, base=10.0))
    w = {k: torch.randn(*s, dtype=torch.float64) for k, s in
         {"q": (H * 2 * d, C), "q.b": (H * 2 * d,), "k": (G * 2 * d, C), "k.b": (G * 2 * d,), "v": (G * dv, C), "v.b": (G * dv,),
          "q.norm": (d,), "k.norm": (d,), "lq1": (d,), "lk1": (d,), "lq2": (d,), "lk2": (d,), "o": (C, H * dv)}.items()}
    h = torch.randn(n, C, dtype=torch.float64)
    got = P.differential_attention(h, w, "", m, eps)

    def prepared(x, wn, t):
        y = [float(v) / math.sqrt(float((x ** 2).mean()) + eps) * float(g) for v, g in zip(x, wn)]
        u, v = y[0], y[1]
        y[0], y[1] = u * math.cos(t) - v * math.sin(t), v * math.cos(t) + u * math.sin(t)
        return y

    lam = math.exp(float(w["lq1"] @ w["lk1"])) - math.exp(float(w["lq2"] @ w["lk2"])) + 0.3
    want = torch.zeros(n, H * dv, dtype=torch.float64)
    for i in range(n):
        qi = (w["q"] @ h[i] + w["q.b"]).view(H, 2, d)
        for a in range(H):
            o = [0.0] * dv
            for t, weight in ((0, 1.0), (1, -lam)):
                es, vs = [], []
                for j in range(max(0, i - size + 1), i + 1):
                    kj = (w["k"] @ h[j] + w["k.b"]).view(G, 2, d)[a // 2, t]
                    s = 0.7 * sum(x * y for x, y in zip(prepared(qi[a, t], w["q.norm"], i), prepared(kj, w["k.norm"], j)))
                    es.append(math.exp(1.5 * math.tanh(s / 1.5)))
                    vs.append((w["v"] @ h[j] + w["v.b"]).view(G, dv)[a // 2])
                for e, v in zip(es, vs):
                    for c in range(dv):
                        o[c] += weight * e / sum(es) * float(v[c])
            r = math.sqrt(sum(x * x for x in o) / dv + eps)
            want[i, a * dv:(a + 1) * dv] = torch.tensor([x / r * 0.7 for x in o], dtype=torch.float64)
    assert float((got - want @ w["o"].T).abs().max()) < 1e-9


def test_plain_latent_attention_and_recurrence_element_by_element():
    import plain_dedunex as P

    torch.manual_seed(1)
    n, C, H, d, r, dv, R, Q, eps = 6, 8, 2, 3, 2, 4, 5, 3, 1e-5
    m = dict(heads=H, dim=d, rot_dim=r, vdim=dv, q_rank=Q, kv_rank=R, scale=0.6, rot=dict(dims=r, base=7.0))
    w = {k: torch.randn(*s, dtype=torch.float64) for k, s in
         {"dq": (Q, C), "dq.norm": (Q,), "uq": (H * (d + r), Q), "dkv": (R + r, C), "dkv.norm": (R,), "uk": (H * d, R),
          "uv": (H * dv, R), "g": (H, C), "o": (C, H * dv)}.items()}
    h = torch.randn(n, C, dtype=torch.float64)
    got = P.latent_attention(h, w, "", m, eps)
    rms = lambda x: x / math.sqrt(float((x ** 2).mean()) + eps)
    turn = lambda x, t: torch.stack([x[0] * math.cos(t) - x[1] * math.sin(t), x[1] * math.cos(t) + x[0] * math.sin(t)])
    want = torch.zeros(n, H * dv, dtype=torch.float64)
    for i in range(n):
        q = (w["uq"] @ (rms(w["dq"] @ h[i]) * w["dq.norm"])).view(H, d + r)
        for a in range(H):
            es, vs = [], []
            for j in range(i + 1):
                kv = w["dkv"] @ h[j]
                c = rms(kv[:R]) * w["dkv.norm"]
                s = float(q[a, :d] @ (w["uk"].view(H, d, R)[a] @ c)) + float(turn(q[a, d:], i) @ turn(kv[R:], j))
                es.append(math.exp(s * 0.6))
                vs.append(w["uv"].view(H, dv, R)[a] @ c)
            gate = 1.0 / (1.0 + math.exp(-float(w["g"][a] @ h[i])))
            want[i, a * dv:(a + 1) * dv] = sum(e * v for e, v in zip(es, vs)) / sum(es) * gate
    assert float((got - want @ w["o"].T).abs().max()) < 1e-9
    # the recurrent unit, one channel at a time
    W = 3
    w = {k: torch.randn(*s, dtype=torch.float64) for k, s in
         {"z": (W, C), "z.b": (W,), "x": (W, C), "x.b": (W,), "g": (W, C), "o": (C, W)}.items()}
    got = P.min_gru(h, w, "")
    sg = lambda v: 1.0 / (1.0 + math.exp(-v))
    want = torch.zeros(n, W, dtype=torch.float64)
    for c in range(W):
        S = 0.0
        for t in range(n):
            z, u, g = sg(float(w["z"][c] @ h[t] + w["z.b"][c])), float(w["x"][c] @ h[t] + w["x.b"][c]), float(w["g"][c] @ h[t])
            S = (1 - z) * S + z * (u + 0.5 if u >= 0 else sg(u))
            want[t, c] = S * g * sg(g)
    assert float((got - want @ w["o"].T).abs().max()) < 1e-9


def test_plain_norm_in_groups_and_the_loops_vectors():
    import plain_dedunex as P

    torch.manual_seed(2)
    x, wt = torch.randn(3, 12, dtype=torch.float64), torch.randn(12, dtype=torch.float64)
    got = P.grouped_norm(x, wt, 3, 1e-3)
    for t in range(3):
        for c in range(12):
            part = x[t, c // 4 * 4:c // 4 * 4 + 4]
            assert abs(float(got[t, c]) - float(x[t, c] / math.sqrt(float((part ** 2).mean()) + 1e-3) * wt[c])) < 1e-12
    assert P.run_order(dict(layers=[0] * 4, loop=dict(start=1, stop=3, times=2))) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert P.run_order(dict(layers=[0] * 2)) == [(0, None), (1, None)]


def _mutations():
    """name -> (change of the configuration, change of the tensors): each is a model that computes one thing wrongly."""
    def at(kind, key, value):
        def change(cfg, w):
            for layer in cfg["layers"]:
                if layer["type"] == kind:
                    d = layer["mixer"]
                    for k in key[:-1]:
                        d = d[k]
                    d[key[-1]] = value(d[key[-1]]) if callable(value) else value
        return change

    def tensor(suffix, f):
        def change(cfg, w):
            for k in list(w):
                if k.endswith(suffix):
                    w[k] = f(w[k])
        return change
    swap = lambda heads: (lambda t: t.view(heads, 2, -1, *t.shape[1:]).flip(1).reshape(t.shape))
    return {
        "a window one position wider": at("attention", ("mask", "size"), lambda v: v + 1),
        "a window one position narrower": at("attention", ("mask", "size"), lambda v: v - 1),
        "no cap on the scores": at("attention", ("softcap",), 0.0),
        "the constant of lambda off": at("attention", ("diff",), lambda v: v + 0.02),
        "no scaled wavelengths": at("attention", ("rot", "scaling"), None),
        "the ramp of the wavelengths elsewhere": at("attention", ("rot", "scaling", "fast"), lambda v: v / 30),
        "fewer turned values": at("attention", ("rot", "dims"), lambda v: v - 2),
        "another base": at("latent_attention", ("rot", "base"), lambda v: v * 1.05),
        "one norm group": lambda cfg, w: cfg["norm"].update(groups=1),
        "another eps": lambda cfg, w: cfg["norm"].update(eps=2e-3),
        "the passes' vectors swapped": tensor("loop.step", lambda t: t.flip(0)),
        "one pass fewer": lambda cfg, w: cfg["loop"].update(times=1),
        "the loop one layer shorter": lambda cfg, w: cfg["loop"].update(stop=2),
        "the maps of a query swapped": tensor("mix.q", swap(4)),
        "the products behind lambda left out": tensor(".lq1", torch.zeros_like),
        "the gates of the latent's heads open": tensor("l1.mix.g", lambda t: t * 0 + 0.0),
        "a gate of another head": tensor("l1.mix.g", lambda t: t.roll(1, 0)),
        "the bias of the values left out": tensor("mix.v.b", torch.zeros_like),
        "the weight of the key norm left out": tensor("mix.k.norm", torch.ones_like),
        "the norm behind the embedding without its weight": tensor("embed.norm", torch.ones_like),
        "update gates a little slower": tensor("mix.z.b", lambda t: t - 0.02),
        "gate and value of the feed-forward swapped": lambda cfg, w: [w.update({p + "gate": w[p + "up"], p + "up": w[p + "gate"]})
                                                                      for p in ("l0.mlp.", "l1.mlp.")],
    }


@pytest.mark.parametrize("name", list(_mutations()))
def test_a_mistake_shows_in_the_logits_of_the_test_models(name, tmp_path):
    """Models that differ from the test model in one mechanism differ in their logits by far more than the bound that the
    comparisons with the engine use."""
    from dedunex_util import TOL, rel_err
    from plain_dedunex import forward, load_folder

    layers = [diff_layer(mlp=dense()), latent_layer(mlp=dense()), gru_layer()]
    cfg, w = load_folder(write_model(config(layers, vocab=90, width=48, loop=(0, 3, 2)), str(tmp_path), seed=4))
    tokens = torch.randint(0, 90, (60,), generator=torch.Generator().manual_seed(1)).tolist()
    right = forward(cfg, w, tokens)
    cfg2, w2 = json.loads(json.dumps(cfg)), dict(w)
    _mutations()[name](cfg2, w2)
    assert rel_err(forward(cfg2, w2, tokens), right) > 20 * TOL["float32"], name

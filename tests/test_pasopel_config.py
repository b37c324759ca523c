"""Pasopel without a GPU: the configuration's reader and its errors, the model as data (parts, tensors, run order, cache
and state needs), pooled rows in the cache manager and the scheduler, and the plain implementation's own checks against
formulas written out element by element."""
import json
import math
import random

import pytest
import torch

from pasopel_util import config, dense, latent_layer, moe, pooled_layer, write_model


def build(cfg_dict):
    from nanoinfer_b200.config import PasopelConfig
    from nanoinfer_b200.models.model import Model
    from nanoinfer_b200.registry import get_architecture

    cfg = PasopelConfig.from_dict(json.loads(json.dumps(cfg_dict)))
    return Model(get_architecture(cfg.architecture).build_spec(cfg), cfg)


def test_the_architecture_is_registered():
    from nanoinfer_b200 import architectures
    from nanoinfer_b200.config.base import architecture_name

    assert {"Pasopel", "Dedunex", "Nagilix", "Kemuzen", "Mulavik", "Vadonex", "GPT2LMHeadModel"} <= set(architectures())
    assert architecture_name({"architecture": "Pasopel"}) == "Pasopel"


def test_all_problems_of_a_configuration_come_in_one_error():
    from nanoinfer_b200.config import ConfigError, PasopelConfig

    bad = config([pooled_layer(heads=3, kv_heads=2), latent_layer(), dict(type="conv", mixer={}), pooled_layer(mlp=dict(kind="gated")),
                  latent_layer(rot_dim=7), pooled_layer(dim=300), pooled_layer(mlp=moe(experts=2, top=3)), pooled_layer(),
                  pooled_layer(), latent_layer(kv_rank=2000)], loop=(2, 99, 0), cap=-1.0)
    del bad["layers"][1]["mixer"]["q_rank"]
    bad["layers"][7]["mixer"]["vdim"] = 5
    bad["layers"][8]["mixer"]["mask"] = dict(size=0, pool=-3)
    bad["norm"].pop("eps")
    with pytest.raises(ConfigError) as e:
        PasopelConfig.from_dict(bad)
    text = str(e.value)
    for piece in ("norm.eps", "logit_softcap", "loop: start 2 and stop 99", "loop.times", "layers[0].mixer.heads",
                  "layers[1].mixer.q_rank", "layers[2].type", "layers[3].mlp.kind", "layers[4].mixer.rot.dims",
                  "layers[5].mixer.dim", "layers[6].mlp.router.top", "layers[7].mixer.vdim", "layers[8].mixer.mask.size",
                  "layers[8].mixer.mask.pool", "layers[9].mixer.kv_rank"):
        assert piece in text, (piece, text)


def test_defaults_of_keys_that_may_be_left_out():
    cfg = config([pooled_layer(conv=0, window=0), latent_layer(rot_dim=0, window=0), pooled_layer(pool=0, mlp=moe(shared=0))], cap=0)
    del cfg["layers"][0]["mixer"]["kv_heads"], cfg["layers"][0]["mixer"]["vdim"]
    m = build(cfg)
    a, lat, b = (blk.mixer for blk in m.layers)
    assert a.n_kv_head == a.n_head and a.window == 0 and a.pool == 0 and not a.conv and a.state_spec() is None
    assert lat.rot_dims == 0 and not lat.halves and lat.element_gate and lat.learned_sink and lat.window == 0
    assert b.window == 24 and b.pool == 0 and m.layers[2].feed_forward.shared_inner == 0
    assert m.stream_vectors is None and m.layers[0].feed_forward is None and m.head.softcap == 0.0
    assert [(e.add_vector, e.add_embedding) for e in m.schedule] == [(None, False)] * 3


def test_run_order_parts_tensors_cache_and_state_of_a_looped_stack():
    from nanoinfer_b200.cache import CacheManager

    layers = [pooled_layer(heads=6, kv_heads=2, dim=20, conv=4, window=24, pool=5, mlp=dense(32)),
              latent_layer(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=20, kv_rank=32, window=9, mlp=moe(5, 2, 24, 16)),
              pooled_layer(heads=2, kv_heads=1, dim=16, conv=1, window=40, pool=16)]
    m = build(config(layers, vocab=99, width=64, loop=(0, 2, 3)))
    assert [(e.layer, e.add_vector, e.add_embedding) for e in m.schedule] == [
        (0, 0, False), (1, None, False), (0, 1, True), (1, None, False), (0, 2, True), (1, None, False), (2, None, False)]
    assert [type(b).__name__ for b in m.layers] == ["PreNormBlock"] * 3 and m.keeps_embedding
    names = {b.ref.name: tuple(b.spec.shape) for b in m.bindings()}
    assert names["loop.step"] == (3, 64) and names["final.norm"] == (64,) and names["embed"] == (99, 64) and "head" not in names
    assert names["l0.mix.q"] == (120, 64) and names["l0.mix.k.b"] == (40,) and names["l0.mix.q.conv"] == (120, 4)
    assert names["l0.mix.g"] == (120, 64) and names["l0.mix.o"] == (64, 120) and names["l0.mix.o.b"] == (64,) and "l0.mix.v" not in names
    assert names["l1.mix.g"] == (72, 64) and names["l1.mix.sink"] == (3,) and names["l1.mix.dkv"] == (40, 64)
    assert names["l1.mlp.router.b"] == (5,) and names["l1.mlp.e4.down"] == (64, 24) and names["l1.mlp.shared.up"] == (16, 64)
    assert names["l0.mlp.up"] == (32, 64) and "l0.mlp.gate" not in names and "l2.norm2" not in names
    kv = dict(m.kv_needs())
    assert set(kv) == {0, 1, 2, 3, 4, 5, 6}                       # every run of a looped layer has pages of its own
    assert (kv[4].n_kv_head, kv[4].head_dim, kv[4].window, kv[4].pool, kv[4].planes) == (2, 32, 24, 5, 2)
    assert (kv[5].head_dim, kv[5].window, kv[5].pool, kv[5].planes) == (40, 9, 0, 1)
    st = dict(m.state_needs())
    assert set(st) == {0, 2, 4} and st[2].shape == (3 * 160,)     # (one tap needs no state)
    cm = CacheManager(m.kv_needs(), m.state_needs(), max_tokens=128, max_requests=2, page_size=16)
    assert len(cm.groups) == 3


def test_stacked_projection_keeps_every_parameter_in_its_place():
    m = build(config([pooled_layer(heads=3, kv_heads=1, dim=10, conv=2, mlp=dense(9)), latent_layer(vdim=5)], width=32))
    g = torch.Generator().manual_seed(0)
    want, per = {}, {}
    for b in m.bindings():
        t = want.setdefault((id(b.part), b.spec.key), torch.randn(b.spec.shape, generator=g))
        per.setdefault(id(b.part), (b.part, {}))[1][b.spec.key] = t.clone()
    for part, params in per.values():
        part.bind(params)
    m.prepare(torch.float32, torch.device("cpu"))
    for b in m.bindings():
        if "norm" in b.where:
            continue                                              # (stored around zero: the one is added at load)
        got = b.part.params[b.spec.key]
        assert torch.equal(got.reshape(b.spec.shape), want[(id(b.part), b.spec.key)]), (b.where, b.spec.key)
    for i, (part, key) in enumerate(((m.layers[0].norm_1, "weight"), (m.final_norm, "weight"))):
        assert torch.equal(part.params[key], want[(id(part), key)] + 1.0)
    a = m.layers[0].mixer
    x = torch.randn(4, 32, generator=g)
    y = x @ a.w_in.T + a.b_in
    assert torch.allclose(y[:, :30], x @ a.params["q_weight"].T + a.params["q_bias"])
    assert torch.allclose(y[:, 30:40], x @ a.params["k_weight"].T + a.params["k_bias"])
    assert torch.allclose(y[:, a.gate_off:a.gate_off + 30], x @ a.params["gate_weight"].T)
    o = torch.randn(4, 3, 16, generator=g)
    assert torch.allclose(o.reshape(4, 48) @ a.w_out.T, o[:, :, :10].reshape(4, 30) @ want[(id(a), "out_weight")].T, atol=1e-5)


# --------------------------------------------------------------------------- pooled rows in the cache
def _manager(window, pool, max_tokens=256, max_requests=3, page=16, **kw):
    from nanoinfer_b200.cache import CacheManager
    from nanoinfer_b200.parts.base import KVCacheSpec

    return CacheManager([(0, KVCacheSpec(2, 16, window, pool=pool)), (1, KVCacheSpec(1, 32, 0))], [], max_tokens=max_tokens,
                        max_requests=max_requests, page_size=page, device=None, **kw)


@pytest.mark.parametrize("window,pool", [(40, 16), (24, 5), (7, 24), (1, 1), (64, 3), (16, 64)])
def test_pages_of_positions_go_back_behind_the_window_and_pooled_rows_stay(window, pool):
    """At every length: what a query or a block that is still to be pooled reads has a page, and so has every pooled row."""
    m = _manager(window, pool, max_tokens=512)
    r = m.open_request()
    while r.n_tokens < 400:
        n = random.Random(r.n_tokens).choice([1, 1, 2, 7, 16, 33])
        m.append([(r, n)])
        end = r.n_tokens + n
        assert len(r.pooled[0]) == -(-(end // pool) // 16) and r.pooled[1] == []
        row, at = r.table_rows[0], m.pool_column[0]
        assert row[at:at + len(r.pooled[0])].tolist() == r.pooled[0] and len(row) == m.max_blocks[0]
        first = min(max(0, r.n_tokens - window + 1), r.n_tokens // pool * pool)
        assert all(r.blocks[0][j // 16] >= 0 for j in range(first, end))
        m.commit(r, n)
        m.check()
    held = sum(1 for p in r.blocks[0] if p >= 0)
    assert held <= (max(window, pool) + 15) // 16 + 2
    m.close_request(r)
    assert m.pages_used() == [0, 0]
    m.check()


def test_a_pool_for_so_many_tokens_takes_a_prompt_of_so_many_tokens_at_once():
    m = _manager(40, 4, max_tokens=256, max_requests=2)
    r = m.open_request()
    assert m.can_append([(r, 256)]) and m.room(r, m.pages_free()) >= 256
    m.append([(r, 256)])
    m.commit(r, 256)
    assert len(r.pooled[0]) == 4 and m.pages_used()[1] == 16
    m.check()


def test_room_is_the_most_that_can_be_appended():
    rnd = random.Random(3)
    for pool in (1, 3, 16, 40):
        m = _manager(16, pool, max_tokens=160, max_requests=2)
        r = m.open_request()
        for _ in range(12):
            free = [rnd.randint(0, f) for f in m.pages_free()]
            n = m.room(r, free)
            fits = lambda k: all(a <= b for a, b in zip(m.pages_needed(r, k), free))
            assert (n == 0 or fits(n)) and not fits(n + 1), (pool, free, n)
            k = rnd.choice([1, 5, 17])
            if m.can_append([(r, k)]):
                m.append([(r, k)])
                m.commit(r, k)


def test_tables_that_grow_keep_both_kinds_of_pages():
    from nanoinfer_b200.cache import CacheManager
    from nanoinfer_b200.parts.base import KVCacheSpec

    m = CacheManager([(0, KVCacheSpec(1, 16, 20, pool=8))], [], max_tokens=64, max_requests=2, page_size=16)
    r = m.open_request()
    gen = m.table_generation
    for _ in range(30):
        m.append([(r, 10)])
        m.commit(r, 10)
        m.check()
    assert m.table_generation > gen and len(r.pooled[0]) == -(-(300 // 8) // 16)
    other = m.open_request()
    m.append([(other, 3)])
    m.check()


def test_truncation_gives_pooled_pages_back():
    m = _manager(4000, 2, max_tokens=512)
    r = m.open_request()
    m.append([(r, 200)])
    m.commit(r, 200)
    assert len(r.pooled[0]) == 7
    m.truncate(r, 70)
    assert len(r.pooled[0]) == 3 and len(r.blocks[0]) == 5
    m.check()


def test_bytes_and_operations_count_the_window_and_the_blocks_behind_it():
    from nanoinfer_b200 import measure

    assert [measure.rows_seen(n, 10, 4) for n in (3, 10, 13, 14, 18, 19)] == [3, 10, 10, 11, 12, 12]
    assert measure.rows_seen(50, 0, 0) == 50 and measure.rows_seen(50, 20, 0) == 20
    m = _manager(10, 4, max_tokens=64)
    m.dtype = torch.float32
    per = 2 * 2 * 16 * 4
    assert measure.kv_bytes(m, [18]) == per * 12 + 2 * 32 * 4 * 18


@pytest.mark.parametrize("seed", range(4))
def test_scheduler_over_pooled_rows_and_a_small_pool(seed):
    """Requests through a pool too small for all of them: portions are cut to the pages that are left, nothing starves, and
    every page comes back."""
    from nanoinfer_b200.engine.scheduler import Scheduler
    from nanoinfer_b200.sampling import SamplingParams
    from test_scheduler import run_step

    rnd = random.Random(seed)
    m = _manager(rnd.choice([16, 40]), rnd.choice([1, 4, 16]), max_tokens=160, max_requests=3)
    s = Scheduler(m, max_batch=3, max_rows=64, prefill_budget=48)
    reqs = [s.add([1] * rnd.randint(1, 110), SamplingParams(max_new_tokens=rnd.randint(1, 30))) for _ in range(7)]
    for _ in range(2000):
        if not s.has_work():
            break
        run_step(m, s)
    assert not s.has_work() and all(r.finish_reason == "length" for r in reqs) and m.pages_used() == [0, 0]


# --------------------------------------------------------------------------- the plain model against written-out formulas
def test_plain_pooled_attention_element_by_element():
    import plain_pasopel as P

    torch.manual_seed(0)
    n, C, H, G, d, taps, size, pool, eps = 23, 10, 4, 2, 4, 3, 6, 4, 1e-5
    m = dict(heads=H, kv_heads=G, dim=d, vdim=d, conv=taps, scale=0.7, mask=dict(size=size, pool=pool))
    w = {k: torch.randn(*s, dtype=torch.float64) for k, s in
         {"q": (H * d, C), "q.b": (H * d,), "k": (G * d, C), "k.b": (G * d,), "q.conv": (H * d, taps), "k.conv": (G * d, taps),
          "sink": (H,), "g": (H * d, C), "o": (C, H * d), "o.b": (C,)}.items()}
    h = torch.randn(n, C, dtype=torch.float64)
    got = P.pooled_window_attention(h, w, "", m, eps)
    up = {x: [w[x] @ h[t] + w[x + ".b"] for t in range(n)] for x in "qk"}
    conv = {x: [sum(w[x + ".conv"][:, j] * up[x][t - taps + 1 + j] for j in range(taps) if t - taps + 1 + j >= 0)
                for t in range(n)] for x in "qk"}
    unit = lambda v: v / math.sqrt(float((v ** 2).mean()) + eps)
    key = lambda t, g: unit(conv["k"][t].view(G, d)[g])
    val = lambda t, g: conv["k"][t].view(G, d)[g]
    want = torch.zeros(n, C, dtype=torch.float64)
    for i in range(n):
        heads = []
        for a in range(H):
            g = a // (H // G)
            pairs = [(key(j, g), val(j, g)) for j in range(n) if 0 <= i - j < size]
            for b in range(n):
                if b * pool + pool - 1 <= i - size:
                    mean = lambda f: sum(f(b * pool + r, g) for r in range(pool)) / pool
                    pairs.append((mean(key), mean(val)))
            qi = unit(conv["q"][i].view(H, d)[a])
            es = [math.exp(0.7 * float(qi @ k)) for k, _ in pairs]
            heads.append(sum(e * v for e, (_, v) in zip(es, pairs)) / (sum(es) + math.exp(float(w["sink"][a]))))
        gate = torch.tensor([1.0 / (1.0 + math.exp(-float(z))) for z in w["g"] @ h[i]], dtype=torch.float64)
        want[i] = w["o"] @ (torch.cat(heads) * gate) + w["o.b"]
    assert float((got - want).abs().max()) < 1e-9


def test_plain_latent_attention_element_by_element():
    import plain_pasopel as P

    torch.manual_seed(1)
    n, C, H, d, r, dv, R, Q, size, eps = 7, 8, 2, 3, 4, 5, 6, 3, 3, 1e-5
    m = dict(heads=H, dim=d, rot_dim=r, vdim=dv, q_rank=Q, kv_rank=R, scale=0.6, rot=dict(dims=r, base=7.0), mask=dict(size=size))
    w = {k: torch.randn(*s, dtype=torch.float64) for k, s in
         {"dq": (Q, C), "dq.norm": (Q,), "uq": (H * (d + r), Q), "dkv": (R + r, C), "dkv.norm": (R,), "uk": (H * d, R),
          "uv": (H * dv, R), "sink": (H,), "g": (H * dv, C), "o": (C, H * dv)}.items()}
    h = torch.randn(n, C, dtype=torch.float64)
    got = P.latent_attention(h, w, "", m, eps)
    rms = lambda x: x / math.sqrt(float((x ** 2).mean()) + eps)

    def turn(x, t):
        y = x.clone()
        for i in range(r // 2):
            a = t * 7.0 ** (-2.0 * i / r)
            y[2 * i] = x[2 * i] * math.cos(a) - x[2 * i + 1] * math.sin(a)
            y[2 * i + 1] = x[2 * i + 1] * math.cos(a) + x[2 * i] * math.sin(a)
        return y
    want = torch.zeros(n, H * dv, dtype=torch.float64)
    for i in range(n):
        q = (w["uq"] @ (rms(w["dq"] @ h[i]) * w["dq.norm"])).view(H, d + r)
        for a in range(H):
            es, vs = [], []
            for j in range(max(0, i - size + 1), i + 1):
                kv = w["dkv"] @ h[j]
                c = rms(kv[:R]) * w["dkv.norm"]
                s = float(q[a, :d] @ (w["uk"].view(H, d, R)[a] @ c)) + float(turn(q[a, d:], i) @ turn(kv[R:], j))
                es.append(math.exp(s * 0.6))
                vs.append(w["uv"].view(H, dv, R)[a] @ c)
            want[i, a * dv:(a + 1) * dv] = sum(e * v for e, v in zip(es, vs)) / (sum(es) + math.exp(float(w["sink"][a])))
        want[i] /= 1.0 + torch.exp(-(w["g"] @ h[i]))
    assert float((got - want @ w["o"].T).abs().max()) < 1e-9


def test_plain_feed_forwards_row_by_row():
    import plain_pasopel as P

    torch.manual_seed(2)
    C, E, F, S, top, n = 6, 4, 3, 5, 2, 7
    w = {k: torch.randn(*s, dtype=torch.float64) for k, s in {"router": (E, C), "router.b": (E,), "shared.gate": (S, C),
                                                              "shared.up": (S, C), "shared.down": (C, S), "up": (F, C), "down": (C, F)}.items()}
    for e in range(E):
        w.update({f"e{e}.gate": torch.randn(F, C, dtype=torch.float64), f"e{e}.up": torch.randn(F, C, dtype=torch.float64),
                  f"e{e}.down": torch.randn(C, F, dtype=torch.float64)})
    h = torch.randn(n, C, dtype=torch.float64)
    got = P.routed_feed_forward(h, w, "", dict(router=dict(experts=E, top=top), shared=dict(ff=S)))
    act = lambda z: z / (1.0 + math.exp(-z))
    gated = lambda p, x: w[p + "down"] @ torch.tensor([act(float(a)) * float(b) for a, b in zip(w[p + "gate"] @ x, w[p + "up"] @ x)],
                                                      dtype=torch.float64)
    for t in range(n):
        z = (w["router"] @ h[t] + w["router.b"]).tolist()
        best = sorted(range(E), key=lambda e: -z[e])[:top]
        total = sum(math.exp(z[e]) for e in best)
        want = gated("shared.", h[t]) + sum(math.exp(z[e]) / total * gated(f"e{e}.", h[t]) for e in best)
        assert float((got[t] - want).abs().max()) < 1e-10
        up = [max(float(v), 0.0) ** 2 for v in w["up"] @ h[t]]
        assert float((P.dense_feed_forward(h, w, "")[t] - w["down"] @ torch.tensor(up, dtype=torch.float64)).abs().max()) < 1e-10


def test_plain_loop_adds_the_embedding_and_the_vectors(tmp_path):
    """Layers without feed-forward, one pass spelled out by hand."""
    import plain_pasopel as P

    cfg, w = P.load_folder(write_model(config([pooled_layer(window=5, pool=2), latent_layer(window=4)], vocab=40, width=32,
                                              loop=(1, 2, 3)), str(tmp_path)))
    tokens = [3, 17, 5, 39, 0, 8, 8, 21, 2, 30, 11]
    got = []
    logits = P.forward(cfg, w, tokens, got)
    w = {k: v.double() for k, v in w.items()}
    norm = lambda x, k: x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + 1e-5) * (1 + w[k])
    x0 = w["embed"][tokens]
    x = x0 + P.pooled_window_attention(norm(x0, "l0.norm1"), w, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5)
    for t in range(3):
        x = x + w["loop.step"][t] + (x0 if t else 0)
        x = x + P.latent_attention(norm(x, "l1.norm1"), w, "l1.mix.", cfg["layers"][1]["mixer"], 1e-5)
        assert float((got[1 + t] - x).abs().max()) < 1e-12
    z = norm(x, "final.norm") @ w["embed"].T
    assert float((logits - 20.0 * torch.tanh(z / 20.0)).abs().max()) < 1e-10


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
            assert any(k.endswith(suffix) for k in w)
            for k in list(w):
                if k.endswith(suffix):
                    w[k] = f(w[k])
        return change

    def patched(name, f):
        return ("patch", name, f)
    import plain_pasopel as P
    keep = {n: getattr(P, n) for n in ("pooled", "softmax_with_sink", "short_conv", "rms")}
    return {
        "a window one position wider": at("attention", ("mask", "size"), lambda v: v + 1),
        "a window one position narrower": at("attention", ("mask", "size"), lambda v: v - 1),
        "the latent's window one wider": at("latent_attention", ("mask", "size"), lambda v: v + 1),
        "blocks one position longer": at("attention", ("mask", "pool"), lambda v: v + 1),
        "no pooled blocks": at("attention", ("mask", "pool"), 0),
        "pooled blocks shifted by one": patched("pooled", lambda x, P_: keep["pooled"](x.roll(1, 0), P_)),
        "the first block empty": patched("pooled", lambda x, P_: torch.cat([0 * keep["pooled"](x, P_)[:1], keep["pooled"](x, P_)[1:]])),
        "sums instead of means": patched("pooled", lambda x, P_: keep["pooled"](x, P_) * P_),
        "no sinks": patched("softmax_with_sink", lambda s, seen, k: keep["softmax_with_sink"](s, seen, k * 0 - 60.0)),
        "sinks of another head": tensor("mix.sink", lambda t: t.roll(1, 0)),
        "no convolution's past": patched("short_conv", lambda x, w: x * w[:, -1]),
        "the taps in the other order": tensor(".conv", lambda t: t.flip(1)),
        "the bias of the keys left out": tensor("mix.k.b", torch.zeros_like),
        "the bias of the output left out": tensor("mix.o.b", torch.zeros_like),
        "gates of another element": tensor("mix.g", lambda t: t.roll(1, 0)),
        "open gates": tensor("mix.g", lambda t: t * 0.0),
        "another base": at("latent_attention", ("rot", "base"), lambda v: v * 1.5),
        "another eps": lambda cfg, w: cfg["norm"].update(eps=2e-2),
        "the passes' vectors swapped": tensor("loop.step", lambda t: t.flip(0)),
        "one pass fewer": lambda cfg, w: cfg["loop"].update(times=1),
        "the loop one layer shorter": lambda cfg, w: cfg["loop"].update(stop=2),
        "no cap on the logits": lambda cfg, w: cfg.update(logit_softcap=None),
        "the router's bias left out": tensor("router.b", torch.zeros_like),
        "one expert more": lambda cfg, w: cfg["layers"][1]["mlp"]["router"].update(top=3),
        "no shared expert": lambda cfg, w: cfg["layers"][1]["mlp"].pop("shared"),
        "norm weights around one": tensor("norm1", lambda t: t - 1.0),
    }


@pytest.mark.parametrize("name", list(_mutations()))
def test_a_mistake_shows_in_the_logits_of_the_test_models(name, tmp_path, monkeypatch):
    """Models that differ from the test model in one mechanism differ in their logits by far more than the bound that the
    comparisons with the engine use."""
    import plain_pasopel as P
    from pasopel_util import TOL, rel_err

    layers = [pooled_layer(heads=4, kv_heads=2, window=17, pool=6, mlp=dense()), latent_layer(mlp=moe()),
              pooled_layer(heads=3, kv_heads=1, window=9, pool=4, mlp=moe(shared=0))]
    cfg, w = P.load_folder(write_model(config(layers, vocab=90, width=48, loop=(0, 3, 2)), str(tmp_path), seed=4))
    tokens = torch.randint(0, 90, (60,), generator=torch.Generator().manual_seed(1)).tolist()
    right = P.forward(cfg, w, tokens)
    cfg2, w2 = json.loads(json.dumps(cfg)), dict(w)
    change = _mutations()[name]
    if isinstance(change, tuple):
        monkeypatch.setattr(P, change[1], change[2])
    else:
        change(cfg2, w2)
    assert rel_err(P.forward(cfg2, w2, tokens), right) > 20 * TOL["float32"], name

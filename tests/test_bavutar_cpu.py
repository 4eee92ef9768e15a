"""Bavutar models without a GPU: configuration, tensor names, sizes that only tensors tell, rejected descriptions, and
checks of the oracle -- each mechanism against an independent form, and that the inputs the GPU tests use show a planted
mistake."""
import ctypes
import json

import numpy as np
import pytest

from oracle import bavutar_oracle as bo
from tests import stack_util as su


@pytest.fixture(scope="module", autouse=True)
def built():
    import __graft_entry__ as ge
    ge.build()


def prepared(cfg, ranks=(7, 5), **over):
    from mesh_transformer import registry
    out = registry.prepare(dict(cfg, **over))
    return registry.family(out).fit_tensors(out, bo.tensor_shapes(cfg, ranks))


@pytest.mark.parametrize("name", sorted(su.BAVUTAR))
def test_tensor_names_and_shapes(name):
    from mesh_transformer import layer_stack, registry
    cfg = prepared(su.BAVUTAR[name], (11, 3))
    registry.family(cfg).validate(cfg)
    assert layer_stack.tensor_shapes(cfg) == bo.tensor_shapes(su.BAVUTAR[name], (11, 3))
    assert registry.prepare(cfg) == cfg


def test_configurations_that_cannot_run_are_rejected():
    from mesh_transformer import registry
    base = su.bavutar([su.gqa(), su.gqa(kv_from=0)])
    bad = [dict(base, cores_per_replica=2), dict(base, loop={"start": 0, "stop": 1, "times": 2}),
           dict(base, layers=[su.gqa(heads=5, kv_heads=2)]), dict(base, layers=[su.ssd(heads=4, groups=3)]),
           dict(base, layers=[su.ssd(heads=4, groups=2, norm_groups=3)]), dict(base, layers=[su.attn()]),
           dict(base, layers=[su.gqa(), su.gqa(kv_from=1)]), dict(base, layers=[su.gqa(), su.gqa(kv_from=0, vdim=8)]),
           dict(base, layers=[su.gqa(), su.gqa(kv_from=0), su.gqa(kv_from=1)]), dict(base, layers=[su.delta(ff=8), su.gqa(kv_from=0)]),
           dict(base, layers=[su.gqa(temp=(0.1, 0))])]
    for cfg in bad:
        with pytest.raises((NotImplementedError, ValueError)):
            registry.family(cfg).validate(prepared(cfg) if cfg["layers"][0]["type"] != "latent_attention" else registry.prepare(cfg))
    with pytest.raises(ValueError, match="decay_rank"):                # sizes that only tensors tell are missing
        registry.family(base).validate(registry.prepare(su.bavutar([su.delta()])))


def test_library_rejects_bad_layers_with_a_message():
    from mesh_transformer import _lib, registry
    caps = dict(rank=0, max_batch=1, max_gen=4, max_rows=32)
    h = ctypes.c_void_p()
    for layers in ([su.gqa(dim=600)], [su.gqa(vdim=0)], [su.delta(dim=300)], [su.ssd(state=300)], [su.ssd(conv=0)], [su.gqa(kv_from=0)]):
        cfg = prepared(su.bavutar(layers))
        assert registry.family(cfg).create(cfg, caps, ctypes.byref(h)) != 0
        assert b"layer 0" in _lib.lib.mtj_last_error()
    for name, model in su.BAVUTAR.items():
        cfg = prepared(model)
        assert registry.family(cfg).create(cfg, caps, ctypes.byref(h)) == 0, name
        assert _lib.lib.mtj_weights_bytes(h) > 0 and _lib.lib.mtj_workspace_bytes(h) > 0
        assert _lib.lib.mtj_destroy(h) == 0


def test_shared_keys_and_values_are_stored_once():
    """A layer that reads another's keys and values adds none to the workspace."""
    from mesh_transformer import _lib, registry
    size = []
    for second in (su.gqa(), su.gqa(kv_from=0)):
        cfg = prepared(su.bavutar([su.gqa(), second]), seq=4096)
        h = ctypes.c_void_p()
        assert registry.family(cfg).create(cfg, dict(rank=0, max_batch=8, max_gen=4, max_rows=32), ctypes.byref(h)) == 0
        size.append(_lib.lib.mtj_workspace_bytes(h))
        _lib.lib.mtj_destroy(h)
    cache = 8 * 4096 * 2 * (24 + 16) * 2                               # slots, positions, key heads, padded columns, bytes
    assert cache <= size[0] - size[1] <= 1.1 * cache


def test_model_folder_round_trip(tmp_path):
    from mesh_transformer import registry
    from mesh_transformer.checkpoint import read_safetensors, write_safetensors
    cfg = su.BAVUTAR["odd"]
    t = su.tensors(su.weights(cfg, 5, ranks=(13, 2)))
    write_safetensors(tmp_path / "model.safetensors", t)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    read = registry.read_config(str(tmp_path), seq=99)
    back = read_safetensors(tmp_path / "model.safetensors")
    fam = registry.family(read)
    fit = fam.fit_tensors(read, {k: tuple(v.shape) for k, v in back.items()})
    assert fit["layers"][0]["mixer"]["decay_rank"] == 13 and fit["layers"][4]["mixer"]["gate_rank"] == 2
    fam.validate(fit)
    assert set(fam.state_from_tensors(fit, back)["layer_stack"]) == set(t)


def test_random_state_has_every_tensor():
    from mesh_transformer import layer_stack, registry
    cfg = prepared(su.BAVUTAR["wide"])
    state = registry.family(cfg).init_state(cfg, 0, "cpu", 1)["params"]["layer_stack"]
    assert {k: tuple(v.shape[1:]) for k, v in state.items()} == layer_stack.tensor_shapes(cfg)
    assert all(bool(v.float().isfinite().all()) for v in state.values())


# ------------------------------------------------------------------- the oracle ----
def test_layer_norm_and_softcap():
    rng = np.random.default_rng(0)
    x = rng.standard_normal((3, 8)) + 5.0
    y = bo.layer_norm(x, 2.0, 1.0, 0.0)
    assert np.allclose(y.mean(-1), 1.0) and np.allclose(y.std(-1), 2.0)
    assert np.allclose(bo.softcap(np.array([1e-4, 1e6, -1e6]), 3.0), [1e-4, 3.0, -3.0]) and bo.softcap(7.0, None) == 7.0


def test_query_temperature_steps():
    t = bo.query_temperature([0, 5, 6, 13, 20], 0.5, 7)
    assert np.allclose(t, 1 + 0.5 * np.log([1, 1, 2, 3, 4]))


def test_grouped_attention_equals_repeated_heads():
    rng = np.random.default_rng(1)
    q, k, v = (rng.standard_normal((9, h, n)) for h, n in ((6, 4), (2, 4), (2, 3)))
    full = bo.causal_attention(q, np.repeat(k, 3, 1), np.repeat(v, 3, 1), 0.7)
    assert np.allclose(bo.causal_attention(q, k, v, 0.7), full)
    s = 0.7 * np.einsum("hn,jhn->hj", q[5], np.repeat(k, 3, 1)[:6])
    w = np.exp(s) / np.exp(s).sum(-1, keepdims=True)
    assert np.allclose(full[5], np.einsum("hj,jhm->hm", w, np.repeat(v, 3, 1)[:6]))


def test_delta_rule_equals_its_product_form():
    """S_t = (I - beta k k^T) diag(g) S_(t-1) + beta k v^T."""
    rng = np.random.default_rng(2)
    T, n, m = 7, 5, 3
    q, k, g = rng.standard_normal((T, 1, n)), bo.unit(rng.standard_normal((T, 1, n))), rng.uniform(0.3, 1, (T, 1, n))
    v, beta = rng.standard_normal((T, 1, m)), rng.uniform(0, 1, (T, 1))
    S = np.zeros((n, m))
    for t in range(T):
        kt = k[t, 0][:, None]
        S = (np.eye(n) - beta[t, 0] * kt @ kt.T) @ np.diag(g[t, 0]) @ S + beta[t, 0] * kt @ v[t, 0][None, :]
    assert np.allclose(bo.delta_rule(q, k, v, g, beta)[-1, 0], S.T @ q[-1, 0])


def test_state_space_dual_equals_its_unrolled_sum():
    rng = np.random.default_rng(3)
    T, H, G, n, m = 8, 4, 2, 5, 3
    x, B, C = rng.standard_normal((T, H, m)), rng.standard_normal((T, G, n)), rng.standard_normal((T, G, n))
    dt, A, D = rng.uniform(0.01, 1, (T, H)), rng.standard_normal(H), rng.standard_normal(H)
    y = bo.state_space_dual(x, B, C, dt, A, D)
    for h in range(H):
        want = D[h] * x[-1, h] + sum(np.exp(-np.exp(A[h]) * dt[s + 1:, h].sum()) * dt[s, h] * (B[s, h // 2] @ C[-1, h // 2]) * x[s, h]
                                     for s in range(T))
        assert np.allclose(y[-1, h], want)


def _changed(cfg, change):
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    return cfg


@pytest.mark.parametrize("fault", ["eps", "alpha", "embed", "cap", "scale", "temp_coef", "temp_every", "kv_from", "norm_groups", "groups"])
def test_random_models_show_a_wrong_constant(fault):
    """The random weights of the GPU tests are such that a wrong constant moves the logits by more than the bf16
    tolerance."""
    cfg = _changed(su.BAVUTAR["odd"], lambda c: c["norm"].update(eps=0.05))
    mix = lambda c, i: c["layers"][i]["mixer"]
    if fault == "kv_from":                                             # layer 3 reads layer 1; here layer 0 has the same sizes
        cfg["layers"][0] = json.loads(json.dumps(cfg["layers"][1]))
    w = su.weights(cfg, 3)
    toks = su.ids(3, 60, cfg["vocab"])
    other = _changed(cfg, {
        "eps": lambda c: c["norm"].update(eps=0.1),
        "alpha": lambda c: c.update(postln_alpha=c["postln_alpha"] * 1.2),
        "embed": lambda c: c["embedding"].update(scale=c["embedding"]["scale"] * 1.3),
        "cap": lambda c: c.update(logit_softcap=3.0),
        "scale": lambda c: mix(c, 1).update(scale=mix(c, 1)["scale"] * 1.3),
        "temp_coef": lambda c: mix(c, 1)["q_temp"].update(coef=0.0),
        "temp_every": lambda c: mix(c, 1)["q_temp"].update(every=20),
        "kv_from": lambda c: mix(c, 3).update(kv_from=0),
        "norm_groups": lambda c: mix(c, 2).update(norm_groups=5),
        "groups": lambda c: (mix(c, 2).update(groups=1, state=27))}[fault])
    assert su.error(bo.forward(other, w, toks), bo.forward(cfg, w, toks)) > 4e-2


@pytest.mark.parametrize("layer", ["delta", "ssd"])
def test_lost_state_shows_long_after(layer):
    cfg = su.bavutar([su.delta() if layer == "delta" else su.ssd()])
    w = su.weights(cfg, 4)
    w["l0.mix.A_log"] = np.full_like(w["l0.mix.A_log"], -4.0)           # slow decays
    toks = su.ids(4, 60, cfg["vocab"])
    assert su.error(bo.forward(cfg, w, toks[30:])[-1:], bo.forward(cfg, w, toks)[-1:]) > 4e-2


def marker_model(heads=4, kv_heads=2, dim=16, vdim=20, temp=None, seed=11):
    """One attention layer in which token 1, as a query, scores token 2's key far above every other key, wherever it
    is: the output shows at once whether that key is seen.  Tokens 3 .. are the background, whose keys are orthogonal to
    the marked query."""
    cfg = su.bavutar([su.gqa(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=1.0, temp=temp, ff=None)], width=64, vocab=40,
                     alpha=1.0, eps=1e-5, scale=1.0, cap=None)
    w = su.weights(cfg, seed)
    rng = np.random.default_rng(seed + 1)
    e = np.linalg.qr(rng.standard_normal((64, 40)))[0].T * 8.0          # orthogonal rows of unit rms
    w["embed"] = bo.to_bf16_grid(e)
    mark = np.sign(rng.standard_normal(dim))
    q, k = rng.standard_normal((40, heads, dim)), rng.standard_normal((40, kv_heads, dim))
    k -= np.einsum("tgn,n->tg", k, mark)[:, :, None] * mark / dim
    q[1], k[2] = mark, mark
    from_embedding = lambda t: bo.to_bf16_grid(np.einsum("tr,td->rd", t.reshape(40, -1), e) / 64.0)
    w["l0.mix.q"], w["l0.mix.k"] = from_embedding(q), from_embedding(k)
    w["l0.mix.v"] = from_embedding(3.0 * rng.standard_normal((40, kv_heads, vdim)))
    w["l0.mix.q.norm"], w["l0.mix.k.norm"] = np.ones_like(w["l0.mix.q.norm"]), np.ones_like(w["l0.mix.k.norm"])
    return cfg, w


def test_marker_model_shows_one_key():
    cfg, w = marker_model()
    toks = 3 + np.arange(300) % 30
    toks[290] = 1
    ref = bo.forward(cfg, w, toks)[290]
    for at in (0, 63, 64, 150, 289):
        seen = toks.copy()
        seen[at] = 2
        assert np.sqrt(np.mean((bo.forward(cfg, w, seen)[290] - ref) ** 2)) > 0.3 * ref.std(), at

"""Kesedra without a GPU: the float64 restatement against itself and against hand-made cases, the
configuration, the weights image, the record tables and packages."""
import ctypes as C
import json

import numpy as np
import pytest

import kesedra_cases as cases
from oracle import kesedra as ref
from smelt_b200 import capi, checkpoint, kesedra, package


# ── the restatement ─────────────────────────────────────────────────────────
def test_rotation_turns_adjacent_pairs():
    x = np.zeros((2, 6))
    x[:, 0], x[:, 3], x[:, 5] = 1.0, 2.0, 7.0
    y = ref.rotate_interleaved(x, [0, 3], 100.0, 4)
    np.testing.assert_allclose(y[0], x[0])
    a, b = 3.0, 3.0 * 100.0 ** -0.5  # pairs 0 and 1
    np.testing.assert_allclose(y[1], [np.cos(a), np.sin(a), -2 * np.sin(b), 2 * np.cos(b), 0, 7.0])


def test_window_and_softmax():
    assert list(ref.window_positions(9, 4)) == [6, 7, 8, 9] and list(ref.window_positions(2, 4)) == [0, 1, 2] and list(ref.window_positions(5, 1)) == [5]
    np.testing.assert_allclose(ref.softmax(np.array([900.0, 900.0 + np.log(3.0)])), [1 / 4, 3 / 4])


def test_latent_scores_are_those_of_the_expanded_keys():
    g = np.random.default_rng(0)
    c, kr, uk, uv = g.standard_normal((7, 5)), g.standard_normal((7, 4)), g.standard_normal((2, 3, 5)), g.standard_normal((2, 6, 5))
    q, qr = g.standard_normal((1, 2, 3)), g.standard_normal((1, 2, 4))
    out = ref.latent_window_attention(q, qr, c, kr, uk, uv, 6, 0.7, 3)
    for h in range(2):
        s = np.array([(uk[h] @ c[j]) @ q[0, h] + kr[j] @ qr[0, h] for j in (4, 5, 6)]) * 0.7
        w = np.exp(s) / np.exp(s).sum()
        np.testing.assert_allclose(out[0, h], sum(w[n] * (uv[h] @ c[j]) for n, j in enumerate((4, 5, 6))))


def test_recurrence_by_hand():
    r, k, v, w, u = (np.array([[[2.0]], [[3.0]]]), np.array([[[5.0]], [[7.0]]]), np.array([[[1.0]], [[-1.0]]]), np.array([[[0.5]], [[0.25]]]), np.array([[10.0]]))
    o, s = ref.wkv(r, k, v, w, u, np.array([[[4.0]]]))
    # first: (4 + 10 * 5) * 2, state 0.5 * 4 + 5; then (7 + 10 * -7) * 3, state 0.25 * 7 - 7
    np.testing.assert_allclose(o[:, 0, 0], [108.0, -189.0])
    np.testing.assert_allclose(s[0, 0, 0], -5.25)


def test_shift_and_decay():
    h = np.arange(6.0).reshape(3, 2)
    np.testing.assert_allclose(ref.token_shift(h, np.array([9.0, 8.0])), [[9, 8], [0, 1], [2, 3]])
    np.testing.assert_allclose(ref.mixed(np.array([[1.0, 1.0]]), np.array([[3.0, 3.0]]), np.array([0.0, 0.5])), [[1.0, 2.0]])
    d = ref.decay(np.array([[2.0]]), np.array([[0.5]]), np.array([[1.0]]), np.array([-1.0]))
    np.testing.assert_allclose(d, np.exp(-np.exp(np.tanh(1.0) - 1.0)))


def test_experts_by_hand():
    eye = np.eye(1)
    f = lambda g, u, limit: ref.expert(np.array([1.0]), g * eye, u * eye, eye, limit)[0]
    gate = lambda g: g / (1 + np.exp(-1.702 * g))
    assert f(2.0, 0.5, 7.0) == pytest.approx(gate(2.0) * 1.5)
    assert f(9.0, -9.0, 7.0) == pytest.approx(gate(7.0) * -6.0)
    assert f(-9.0, 9.0, 7.0) == pytest.approx(gate(-9.0) * 8.0)  # the gate has no lower limit
    chosen, weights = ref.route(np.ones((1, 1)), np.array([[1.0], [3.0], [2.0]]), np.array([0.0, 0.0, 2.0]), 2)
    assert chosen.tolist() == [[2, 1]]
    np.testing.assert_allclose(weights, [[np.e / (1 + np.e), 1 / (1 + np.e)]])


def test_norms():
    x = np.array([3.0, 4.0])
    np.testing.assert_allclose(ref.zero_centred_norm(x, np.array([0.0, 1.0]), 0.5), np.array([3.0, 8.0]) / np.sqrt(13.0))
    np.testing.assert_allclose(ref.plain_norm(x, np.array([0.0, 1.0]), 0.5), np.array([0.0, 4.0]) / np.sqrt(13.0))


@pytest.mark.parametrize("name", cases.ALL)
def test_restatement_in_portions_equals_whole(name):
    cfg = cases.ALL[name]
    m = ref.Kesedra(cfg, cases.tensors(cfg))
    toks = cases.tokens(cfg, 60)
    whole = m.feed(toks)
    m.reset()
    parts = [m.feed(toks[a:b]) for a, b in ((0, 1), (1, 3), (3, 40), (40, 41), (41, 60))]
    np.testing.assert_allclose(np.concatenate(parts), whole, rtol=1e-9, atol=1e-9)


@pytest.mark.parametrize("name", cases.ALL)
def test_the_cases_have_no_close_choices(name):
    cfg = cases.ALL[name]
    t = cases.tensors(cfg)
    assert cases.close_calls(cfg, t, ref.Kesedra(cfg, t), cases.tokens(cfg, 150), 0.04) == 0.0


# ── configuration ───────────────────────────────────────────────────────────
def test_parse_reads_every_size():
    c = kesedra.parse(cases.MIXED)
    a, b = c.layers[1].mixer, c.layers[2].mixer
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank, a.q_rank, a.window, a.kv_from, a.rot_base, a.rot_dims) == (4, 32, 16, 48, 40, 56, 24, -1, 1000.0, 16)
    assert (b.kv_from, b.scale) == (1, 0.3) and c.layers[0].mixer == kesedra.WkvConfig(3, 32) and c.layers[3].mlp is None
    assert c.layers[2].mlp == kesedra.ExpertsConfig(24, 0.4, 9, 3) and c.layers[1].mlp == kesedra.DenseConfig(160)
    shapes = kesedra.tensor_shapes(c, lambda i: 24)
    assert "l2.mix.dkv" not in shapes and shapes["l1.mix.dkv"] == (56, 96) and "l3.norm2" not in shapes and shapes["l2.mlp.e8.down"] == (96, 24) and shapes["l3.mix.w1"] == (24, 96)


@pytest.mark.parametrize("edit", [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][1]["mlp"].update(kind="gated"), lambda c: c.pop("norm"),
                                  lambda c: c["layers"][1]["mixer"]["mask"].pop("size"), lambda c: c["layers"][0]["mixer"].update(heads=0), lambda c: c["layers"][2]["mixer"].update(kv_from=4),
                                  lambda c: c["layers"][2]["mixer"].update(kv_from=0), lambda c: c["layers"][5]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(kv_rank=64),
                                  lambda c: c["layers"][2]["mixer"]["rot"].update(base=7.0), lambda c: c["layers"][0]["mlp"]["router"].update(top=7), lambda c: c.update(layers=[])])
def test_unknown_or_incomplete_configurations_are_refused(edit):
    c = json.loads(json.dumps(cases.MIXED))
    edit(c)
    with pytest.raises(checkpoint.CheckpointError):
        checkpoint.architecture(c).parse(c)


def test_registry_knows_the_design():
    assert "Kesedra" in checkpoint.architectures()


def test_missing_and_misshapen_tensors_are_refused():
    t = cases.stored(cases.tensors(cases.ODD))
    c = kesedra.parse(cases.ODD)
    for name, other in (("l0.mix.uk", None), ("l1.mix.w1", None), ("head", ("BF16", t["head"][1][:, :-1])), ("l3.mlp.e34.gate", ("F32", t["l3.mlp.e34.gate"][1].astype(np.float32)))):
        broken = {k: v for k, v in t.items() if k != name} | ({name: other} if other else {})
        with pytest.raises(checkpoint.CheckpointError, match=name):
            kesedra.build_image(c, checkpoint.TensorFile(broken))


def test_image_holds_the_joined_and_padded_matrices():
    cfg, t = cases.MIXED, cases.tensors(cases.MIXED)
    image, desc, layers, entries = kesedra.build_image(kesedra.parse(cfg), checkpoint.TensorFile(cases.stored(t)))

    def tensor(off, *shape):
        assert off % 128 == 0
        return checkpoint.bf16_to_f32(image[off:off + int(np.prod(shape)) * 2].view(np.uint16)).reshape(shape)

    w = tensor(layers[0].in_proj, 4 * 128 + 64, 128)  # r, k, v, g of 96 rows in groups of 128, then the decay's 24
    for n, s in enumerate("rkvg"):
        np.testing.assert_array_equal(w[128 * n:128 * n + 96, :96], t[f"l0.mix.{s}"])
        assert not w[128 * n + 96:128 * n + 128].any()
    np.testing.assert_array_equal(w[512:536, :96], t["l0.mix.w1"])
    assert not w[536:].any() and not w[:, 96:].any()
    np.testing.assert_array_equal(tensor(layers[0].mu, 5, 128)[4, :96], t["l0.mix.mu.w"])
    up = tensor(layers[0].up, 6, 64, 2, 128)
    np.testing.assert_array_equal(up[5, :40, 0, :96], t["l0.mlp.e5.gate"])
    np.testing.assert_array_equal(up[5, :40, 1, :96], t["l0.mlp.e5.up"])
    assert not up[:, 40:].any()
    w = tensor(layers[1].in_proj, 64 + 40 + 16, 128)
    np.testing.assert_array_equal(w[:56, :96], t["l1.mix.dq"])
    np.testing.assert_array_equal(w[64:, :96], t["l1.mix.dkv"])
    assert not w[56:64].any()
    q = tensor(layers[2].q_proj, 2, 32 + 16, 128)  # heads of 24 + 16 rows, padded to 32 + 16
    uq = t["l2.mix.uq"].reshape(2, 40, 72)
    np.testing.assert_array_equal(q[:, :24, :72], uq[:, :24])
    np.testing.assert_array_equal(q[:, 32:, :72], uq[:, 24:])
    assert not q[:, 24:32].any()
    kv = tensor(layers[1].kv_proj, 4 * 32 + 4 * 64, 64)
    np.testing.assert_array_equal(kv[:128, :40], t["l1.mix.uk"])
    np.testing.assert_array_equal(kv[128:].reshape(4, 64, 64)[:, :48, :40], t["l1.mix.uv"].reshape(4, 48, 40))
    np.testing.assert_array_equal(tensor(layers[1].out_proj, 96, 4, 64)[:, :, :48], t["l1.mix.o"].reshape(96, 4, 48))
    freq = image[layers[1].rot_freq:layers[1].rot_freq + 64].view(np.float64)
    np.testing.assert_allclose(freq, 1000.0 ** (-np.arange(8) / 8))
    assert layers[2].kv_from == 1 and layers[1].kv_from == -1 and layers[3].ff_kind == capi.FF_NONE
    assert {e[0] for e in entries} >= {"embed", "head", "l2.mix.ukv", "l0.mlp.gate_up", "final.norm"}


# ── record tables ───────────────────────────────────────────────────────────
def build(name):
    cfg = cases.ALL[name]
    _, desc, layers, _ = kesedra.build_image(kesedra.parse(cfg), checkpoint.TensorFile(cases.stored(cases.tensors(cfg))))
    return desc, layers


def count(b, prefill):
    n = C.c_size_t(0)
    return b.table(prefill)[1](None, None, C.byref(n)), n.value


@pytest.mark.parametrize("name,state", [("mixed", 8), ("odd", 8), ("wide", 8)])
def test_tables_cover_the_layers(name, state):
    desc, layers = build(name)
    b = package.DenseBuilders(desc, layers, 600, 64)
    c = kesedra.parse(cases.ALL[name])
    decode = {True: 6, False: 3}  # launches of a mixer: latent attention, time mixing
    ff = {type(None): 0, kesedra.DenseConfig: 2, kesedra.ExpertsConfig: 3}
    sublayers = sum(1 + (layer.mlp is not None) for layer in c.layers)
    want = 1 + sum(decode[isinstance(layer.mixer, kesedra.LatentConfig)] + ff[type(layer.mlp)] for layer in c.layers) + (sublayers - 1) + 3  # a swap for every sublayer read in front of another
    assert count(b, False) == (0, want)
    assert count(b, True)[0] == 0
    assert len(b.cache_slots()) == state
    sizes = dict(b.slots())
    if name == "mixed":  # the ring holds the longest window that reads it, and a chunk
        owner = b.cache_slots()[2]
        assert sizes[owner] == -(-(37 + 64) // 64) * 64 * 64 * 2


def test_table_builder_refuses_bad_descriptions():
    for edit in (lambda w: setattr(w[1], "window", 0), lambda w: setattr(w[2], "kv_from", 2), lambda w: setattr(w[2], "kv_from", 0), lambda w: setattr(w[0], "top", 7), lambda w: setattr(w[0], "mixer", 5)):
        desc, layers = build("mixed")
        edit(layers)
        for prefill in (False, True):
            assert count(package.DenseBuilders(desc, layers, 600, 64), prefill)[0] == capi.BAD_ARGUMENT


def test_kernel_names_are_bound():
    lib = capi.load()
    for name in ("smelt_embed_rows", "smelt_matvec:64:64", "smelt_matvec_shift:128:96", "smelt_matvec_experts_in:128:96", "smelt_latent_scores_bf16:120:56", "smelt_latent_prefill_bf16:64:64",
                 "smelt_wkv_decode", "smelt_wkv_gate_rows_f32", "smelt_dense_gemm_groups_bf16:128:128", "smelt_expert_gemm_glu_f32:64:64", "smelt_moe_combine:64:64", "smelt_residual_norm_rows_bf16"):
        assert lib.smelt_cuda_pipeline_supported(name.encode()) == 1, name
    assert lib.smelt_cuda_pipeline_supported(b"smelt_latent_scores_fp8:64:64") == 0


@pytest.mark.parametrize("name", cases.ALL)
def test_package_of_the_model_validates(tmp_path, name):
    cfg, folder, out = cases.ALL[name], tmp_path / "model", tmp_path / "x.smeltpkg"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    checkpoint.write_safetensors(str(folder / "model.safetensors"), cases.stored(cases.tensors(cfg)))
    checkpoint.convert(str(folder), str(out), max_chunk=64)
    st, info, err = package.inspect_package(str(out))
    assert st == 0, err
    assert info.vocab_size == cfg["vocab"] and info.n_prefill_records > 0
    manifest = json.loads((out / "manifest.json").read_text())
    assert sum(s["category"] == "state" for s in manifest["buffers"]["slots"]) == 8
    assert all(e["offset"] % 128 == 0 for e in manifest["weights"]["entries"])

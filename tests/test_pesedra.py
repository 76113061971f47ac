"""Pesedra without a GPU: the float64 restatement against itself and against hand-made cases, model
folders, the weights image, the record tables, and the trace replay's bookkeeping."""
import ctypes as C
import json

import numpy as np
import pytest

import pesedra_cases as cases
from oracle import pesedra as ref
from smelt_b200 import capi, checkpoint, generate, package, pesedra, trace_run


# ── the restatement ─────────────────────────────────────────────────────────
def test_visible_keys():
    # window 4: positions 6..9 at 9; pool 3: a block once its last position is four back
    assert list(ref.window_positions(9, 4)) == [6, 7, 8, 9]
    assert list(ref.window_positions(2, 4)) == [0, 1, 2]
    assert [ref.pooled_blocks(i, 4, 3) for i in (5, 6, 8, 9, 11, 12)] == [[], [0], [0], [0, 1], [0, 1], [0, 1, 2]]
    assert ref.pooled_blocks(3, 1, 1) == [0, 1, 2]


def test_sink_softmax_adds_one_to_the_denominator():
    s = np.array([0.0, np.log(2.0)])
    np.testing.assert_allclose(ref.sink_softmax(s), [1 / 4, 2 / 4])
    np.testing.assert_allclose(ref.sink_softmax(np.array([-50.0])), [np.exp(-50.0) / (1 + np.exp(-50.0))])
    assert ref.sink_softmax(np.array([800.0]))[0] == pytest.approx(1.0)


def test_xielu_branches():
    p, q = 0.3, -0.7
    sp, sq = np.log(1 + np.exp(p)), np.log(1 + np.exp(q))
    z = np.array([2.0, -1.5, 0.0])
    np.testing.assert_allclose(ref.xielu(z, p, q), [sp * 4 + 1, (0.5 + sq) * (np.exp(-1.5) - 1 + 1.5) - 0.75, 0.0])


def test_block_mean_and_grouped_heads():
    g = np.random.default_rng(0)
    q, k, v = g.standard_normal((1, 4, 8)), g.standard_normal((12, 2, 8)), g.standard_normal((12, 2, 6))
    out = ref.window_pool_attention(q, k, v, 11, 0.5, 7.0, 4, 3)
    for h in range(4):
        keys = np.concatenate([k[8:12, h // 2], [k[0:3, h // 2].mean(0), k[3:6, h // 2].mean(0)]])
        vals = np.concatenate([v[8:12, h // 2], [v[0:3, h // 2].mean(0), v[3:6, h // 2].mean(0)]])
        e = np.exp(7.0 * np.tanh(keys @ q[0, h] * 0.5 / 7.0))
        np.testing.assert_allclose(out[0, h], e @ vals / (1 + e.sum()))


def test_layer_runs():
    assert ref.layer_runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert ref.layer_runs({"layers": [0] * 2}) == [(0, False), (1, False)]


@pytest.mark.parametrize("name", cases.ALL)
def test_restatement_in_portions_equals_whole(name):
    cfg = cases.ALL[name]
    m = ref.Pesedra(cfg, cases.tensors(cfg))
    toks = cases.tokens(cfg, 70)
    whole = m.feed(toks)
    m.reset()
    parts = [m.feed(toks[a:b]) for a, b in ((0, 1), (1, 3), (3, 40), (40, 41), (41, 70))]
    np.testing.assert_allclose(np.concatenate(parts), whole, rtol=1e-9, atol=1e-9)


# ── model folders and configuration ─────────────────────────────────────────
def test_safetensors_round_trip(tmp_path):
    t = {"a": ("BF16", np.arange(6, dtype=np.uint16).reshape(2, 3)), "s": ("BF16", np.array(0x3F80, np.uint16)), "i": ("I32", np.arange(4, dtype=np.int32))}
    checkpoint.write_safetensors(str(tmp_path / "m.safetensors"), t)
    back = checkpoint.read_safetensors(str(tmp_path / "m.safetensors"))
    assert {k: (d, a.tolist()) for k, (d, a) in back.items()} == {k: (d, a.tolist()) for k, (d, a) in t.items()}
    wide = ref.read_safetensors(str(tmp_path / "m.safetensors"))
    assert wide["s"] == 1.0 and wide["s"].shape == ()


def test_bf16_rounding_is_to_nearest_even():
    a = np.array([1.0, 1.0 + 2 ** -8, 1.0 + 3 * 2 ** -8, -3.14159], np.float32)
    np.testing.assert_array_equal(cases.round_bf16(a), np.array([1.0, 1.0, 1.0 + 2 ** -6, -3.140625], np.float32))


def test_parse_reads_every_size():
    c = pesedra.parse(cases.MIXED)
    assert c.runs() == [0, 1, 2, 1, 2, 1, 2, 3] and c.layers[1].ff == 0 and c.layers[2].scale == 0.3 and c.layers[0].vdim == 48
    assert pesedra.parse(cases.ODD).loop == (0, 0, 0)
    assert "loop.in" not in pesedra.tensor_shapes(pesedra.parse(cases.ODD))
    assert "l1.mlp.up" not in pesedra.tensor_shapes(c) and pesedra.tensor_shapes(c)["l0.mix.o"] == (96, 192)


@pytest.mark.parametrize("edit", [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="gated"), lambda c: c.pop("norm"),
                                  lambda c: c["layers"][0]["mixer"]["mask"].pop("pool"), lambda c: c["layers"][0]["mixer"].update(heads=5),
                                  lambda c: c["loop"].update(stop=9), lambda c: c.update(architecture="Unheard")])
def test_unknown_or_incomplete_configurations_are_refused(edit):
    c = json.loads(json.dumps(cases.MIXED))
    edit(c)
    with pytest.raises(checkpoint.CheckpointError):
        checkpoint.architecture(c).parse(c)


def test_registry_knows_the_design():
    assert "Pesedra" in checkpoint.architectures()


def test_missing_and_misshapen_tensors_are_refused():
    t = cases.stored(cases.tensors(cases.ODD))
    c = pesedra.parse(cases.ODD)
    for name, other in (("l0.mix.k", None), ("head", ("BF16", t["head"][1][:, :-1])), ("pos", ("F32", t["pos"][1].astype(np.float32)))):
        broken = {k: v for k, v in t.items() if k != name} | ({name: other} if other else {})
        with pytest.raises(checkpoint.CheckpointError, match=name):
            pesedra.build_image(c, checkpoint.TensorFile(broken))


def test_image_holds_the_joined_and_padded_matrices():
    cfg, t = cases.MIXED, cases.tensors(cases.MIXED)
    c = pesedra.parse(cfg)
    image, desc, layers = pesedra.build_image(c, checkpoint.TensorFile(cases.stored(t)))

    def matrix(off, rows, cols):
        assert off % 128 == 0
        return checkpoint.bf16_to_f32(image[off:off + rows * cols * 2].view(np.uint16)).reshape(rows, cols)

    joined = np.concatenate([t["l0.mix.q"], t["l0.mix.k"], t["l0.mix.v"], t["l0.mlp.up"]])
    w = matrix(layers[0].in_proj, joined.shape[0], 128)
    np.testing.assert_array_equal(w[:, :96], joined)
    assert not w[:, 96:].any()
    out = np.concatenate([t["l0.mix.o"], t["l0.mlp.down"]], 1)
    w = matrix(layers[0].out_proj, 96, 384)
    np.testing.assert_array_equal(w[:, :352], out)
    assert not w[:, 352:].any()
    w = matrix(desc.loop_in, 96, 256)
    np.testing.assert_array_equal(w[:, :96], t["loop.in"][:, :96])
    np.testing.assert_array_equal(w[:, 128:224], t["loop.in"][:, 96:])
    assert layers[1].ff == 0 and desc.final_gain == t["final.norm"]
    assert layers[0].act_falling == pytest.approx(0.5 + np.log1p(np.exp(t["l0.mlp.act"][1])))


# ── record tables ───────────────────────────────────────────────────────────
def count(fn, desc, layers, capacity=600, chunk=64):
    n = C.c_size_t(0)
    st = fn(None, C.byref(desc), layers, capacity, chunk, None, C.byref(n))
    return st, n.value


def test_table_sizes_follow_the_layer_runs():
    lib = capi.load()
    for cfg, runs, passes in ((cases.MIXED, 8, 3), (cases.ODD, 2, 0), (cases.WIDE, 4, 2)):
        _, desc, layers = pesedra.build_image(pesedra.parse(cfg), checkpoint.TensorFile(cases.stored(cases.tensors(cfg))))
        assert count(lib.smelt_cuda_build_dense_decoder, desc, layers) == (0, 1 + 3 * runs + 2 * passes + 3)  # a swap beside every entry projection
        assert count(lib.smelt_cuda_build_dense_prefill_table, desc, layers) == (0, 1 + 6 * runs + 2 * passes + 4)
        first, n = C.c_int32(), C.c_int32()
        assert lib.smelt_cuda_dense_cache_slots(C.byref(desc), C.byref(first), C.byref(n)) == 0 and n.value == 2 * runs


def test_table_builder_refuses_bad_descriptions():
    lib = capi.load()
    _, desc, layers = pesedra.build_image(pesedra.parse(cases.ODD), checkpoint.TensorFile(cases.stored(cases.tensors(cases.ODD))))
    assert count(lib.smelt_cuda_build_dense_decoder, desc, layers, capacity=641)[0] == capi.BAD_ARGUMENT  # past the position table
    layers[0].pool = 0
    assert count(lib.smelt_cuda_build_dense_decoder, desc, layers)[0] == capi.BAD_ARGUMENT


def test_dense_kernel_names_are_bound():
    lib = capi.load()
    for name in ("smelt_embed_positions", "smelt_dense_matvec:128:96", "smelt_dense_matvec_xielu:64:64", "smelt_dense_matvec_add:64:64", "smelt_window_decode_bf16", "smelt_window_pool_f32",
                 "smelt_dense_gemm_bf16:64:64", "smelt_dense_gemm_add_f32:64:64", "smelt_window_attention_f32:64:64", "argmax_f32_partials"):
        assert lib.smelt_cuda_pipeline_supported(name.encode()) == 1, name
    assert lib.smelt_cuda_pipeline_supported(b"smelt_window_decode_fp8") == 0


@pytest.mark.parametrize("name", cases.ALL)
def test_package_of_the_model_validates(tmp_path, name):
    cfg, folder, out = cases.ALL[name], tmp_path / "model", tmp_path / "x.smeltpkg"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    checkpoint.write_safetensors(str(folder / "model.safetensors"), cases.stored(cases.tensors(cfg)))
    checkpoint.convert(str(folder), str(out), max_chunk=64)
    st, info, err = package.inspect_package(str(out))
    assert st == 0, err
    runs = len(pesedra.parse(cfg).runs())
    assert info.vocab_size == cfg["vocab"] and info.n_prefill_records > 6 * runs and info.n_records > 3 * runs
    manifest = json.loads((out / "manifest.json").read_text())
    assert sum(s["category"] == "state" for s in manifest["buffers"]["slots"]) == 2 * runs
    assert all(e["offset"] % 128 == 0 for e in manifest["weights"]["entries"])


# ── trace replay ────────────────────────────────────────────────────────────
class FakeDecoder:
    def __init__(self):
        self.calls = []

    def feed(self, tokens, start, want):
        self.calls.append((list(tokens), start, list(want)))
        return np.array([[tokens[w], start + w] for w in want], np.float32).reshape(len(want), 2)


def test_replay_follows_one_sequence_at_a_time():
    d = FakeDecoder()
    r = trace_run.Replay(d)
    out = r.step([{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}], [])
    np.testing.assert_array_equal(out, [[5, 0], [7, 2]])
    assert r.step([{"id": "a", "tokens": [8], "want": []}], ["a"]).shape == (0, 2)
    np.testing.assert_array_equal(r.step([{"id": "b", "tokens": [9], "want": [0]}], []), [[9, 0]])
    assert d.calls == [([5, 6, 7], 0, [0, 2]), ([8], 3, []), ([9], 0, [0])]
    with pytest.raises(ValueError, match="live"):
        r.step([{"id": "c", "tokens": [1], "want": []}], [])


def test_prompt_ids(tmp_path):
    (tmp_path / "ids").write_text("4, 5\n6")
    assert generate.parse_ids("1,2,3") == [1, 2, 3] and generate.parse_ids(f"@{tmp_path / 'ids'}") == [4, 5, 6]

"""CPU checks of the layer-list models' host side: configuration and registry, safetensors files, rotation tables and the
bigram hash against the oracle, the request queue and the trace replay over a stand-in decoder, argument validation of the C ABI."""
import ctypes as C
import io
import json
import os
import re

import numpy as np
import pytest
import torch

from cut_b200 import _lib as L
from cut_b200 import bigerax, models
from cut_b200.decoding import RequestQueue, generate
from cut_b200.layer_list import GatedRecurrence, LayerListDecoder, Rotation, WindowAttention, rotation_tables
from cut_b200.safetensors_io import SafetensorsFile, write_safetensors
from oracle import hybrid_ref as R
from tests.layer_list_util import CONFIGS, attention, config, mingru, random_weights, save_model, torch_weights, with_mlp

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_configuration_reads_every_size_and_constant():
    c = bigerax.parse_config(CONFIGS["gqa"])
    assert (c.width, c.vocab, c.norm_groups, c.norm_eps, len(c.layers)) == (96, 203, 3, 1e-6, 6)
    assert (c.bigram.buckets, c.bigram.mul_prev, c.bigram.mul_cur) == (53, 7, 5)
    a = c.layers[0].mixer
    assert isinstance(a, WindowAttention) and (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.rot.dims, a.rot.base) == (6, 2, 40, 24, 33, 16, 10000.0)
    assert a.sink and a.v_mix and not c.layers[4].mixer.v_mix and c.first_mixing == 0
    assert c.layers[1].mlp is None and c.layers[3].mlp.ff == 56 and c.layers[3].mixer == GatedRecurrence(130)
    assert bigerax.parse_config(CONFIGS["odd"]).first_mixing == 1
    assert bigerax.parse_config(config(8, 9, [with_mlp(mingru(4), 0)])).first_mixing == -1


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0].update(type="mystery"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="mystery"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rotated elements"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "empty window"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=48), "same value heads"),
    (lambda c: c["norm"].update(groups=5), "divide the width"),
])
def test_configuration_refuses_what_it_does_not_know(change, what):
    c = json.loads(json.dumps(CONFIGS["gqa"]))
    change(c)
    with pytest.raises(ValueError, match=what):
        bigerax.parse_config(c)


def test_registry_finds_the_model_by_its_own_files(tmp_path):
    w = random_weights(CONFIGS["odd"], 1)
    folder = save_model(tmp_path / "m", CONFIGS["odd"], w)
    entry, cfg = models.read_config(folder)
    assert entry.decoder is LayerListDecoder and cfg.vocab == 99 and "float32" in entry.dtypes
    f = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    g = entry.gather_weights(cfg, f.get, f.__contains__)
    assert torch.equal(g["layers"][1]["mix"]["k"].float(), torch.from_numpy(w["l1.mix.k"])) and "g.b" not in g["layers"][0]["mix"]
    assert g["layers"][2]["mix"]["vmix"] == float(w["l2.mix.vmix"]) and "vmix" not in g["layers"][1]["mix"]
    with open(os.path.join(folder, "config.json"), "w") as fh:
        json.dump({"architecture": "Nothing"}, fh)
    with pytest.raises(ValueError, match="unknown architecture"):
        models.read_config(folder)


def test_safetensors_round_trip_and_refusals(tmp_path):
    p = str(tmp_path / "t.safetensors")
    t = {"a": torch.arange(12, dtype=torch.float32).reshape(3, 4), "s": torch.tensor(1.5, dtype=torch.bfloat16),
         "i": torch.tensor([1, -2, 3], dtype=torch.int32), "b": torch.randn(5, 3).to(torch.bfloat16)}
    write_safetensors(p, t)
    f = SafetensorsFile(p)
    assert sorted(f.names()) == sorted(t) and "a" in f and "z" not in f
    for k, v in t.items():
        assert f.get(k).dtype == v.dtype and f.get(k).shape == v.shape and torch.equal(f.get(k), v)
    with pytest.raises(KeyError):
        f.get("z")
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-4])
    with pytest.raises(ValueError, match="does not fit"):
        SafetensorsFile(p)
    open(p, "wb").write(b"\xff\xff\xff\xff\x00\x00\x00\x00{}")
    with pytest.raises(ValueError, match="header length"):
        SafetensorsFile(p)


def test_rotation_tables_are_the_oracles_rotation():
    rot = Rotation(500.0, 12)
    c, s = rotation_tables(rot, 40)
    x = np.random.default_rng(0).standard_normal((40, 2, 20))
    want = R.rotate_pairs(x, np.arange(40), rot.base, rot.dims)
    got = x.copy()
    a, b = x[:, :, 0:12:2], x[:, :, 1:12:2]
    got[:, :, 0:12:2], got[:, :, 1:12:2] = a * c[:, None] - b * s[:, None], b * c[:, None] + a * s[:, None]
    assert np.abs(got - want).max() < 1e-6 and np.array_equal(want[:, :, 12:], x[:, :, 12:])


def test_oracle_mechanisms_on_hand_sized_cases():
    # a window of 2 with one key far above the others: it is seen for two positions and then never again
    k = np.zeros((6, 1, 2))
    k[1, 0, 0] = 100.0
    v = np.arange(6.0).reshape(6, 1, 1)
    q = np.ones((6, 1, 2))
    out = R.window_attention(q, k, v, 0, 2, 1.0)
    assert abs(out[1, 0] - 1.0) < 1e-12 and abs(out[2, 0] - 1.0) < 1e-12 and abs(out[4, 0] - (3 + 4) / 3) < 1e-12
    assert list(R.bigram_rows([4, 2], None, 7, 5, 53)) == [53, (4 * 7 + 2 * 5) % 53] and list(R.bigram_rows([2], 4, 7, 5, 53)) == [38]
    s = R.mingru_scan(np.array([[0.5], [1.0]]), np.array([[1.0], [0.0]]), np.array([2.0]))
    assert np.allclose(s[:, 0], [0.5 * 2 + 0.5 * 1.5, 0.5])
    x = np.array([3.0, 4.0, 0.0, 2.0])
    assert np.allclose(R.grouped_norm(x, np.ones(4), 2, 0.0), [3 / np.sqrt(12.5), 4 / np.sqrt(12.5), 0.0, np.sqrt(2.0)])


def test_oracle_continues_a_sequence_at_any_cut():
    cfg = CONFIGS["gqa"]
    ref = R.HybridReference(cfg, random_weights(cfg, 3))
    toks = np.random.default_rng(5).integers(0, cfg["vocab"], 50)
    whole = ref.run(toks)
    ref.reset()
    parts = np.concatenate([ref.run(toks[a:b]) for a, b in ((0, 1), (1, 3), (3, 40), (40, 50))])
    assert np.abs(whole - parts).max() < 1e-10


class FakeDecoder:
    """Counts upwards from the sum of what it was fed."""

    def __init__(self, slots=1):
        self.free, self.calls = slots, []

    def open(self):
        if not self.free:
            raise RuntimeError("no free sequence place")
        self.free -= 1
        return {"sum": 0}

    def close(self, s):
        self.free += 1

    def forward(self, s, tokens, want):
        rows = []
        for i, t in enumerate(tokens):
            s["sum"] += t
            if i in want:
                rows.append([s["sum"], -s["sum"]])
        self.calls.append((list(tokens), list(want)))
        return torch.tensor(rows, dtype=torch.float32) if rows else None

    def decode_greedy(self, s, n):
        return [s["sum"] + i for i in range(n)]

    def check_status(self):
        pass


def test_request_queue_serves_in_order_and_cuts_prompts():
    d = FakeDecoder()
    q = RequestQueue(d, portion=2)
    a, b = q.submit([1, 2, 3, 4, 5], 2), q.submit([7], 3)
    q.run()
    assert a.tokens == [15, 16] and b.tokens == [7, 8, 9] and d.free == 1
    assert d.calls == [([1, 2], []), ([3, 4], []), ([5], [0]), ([7], [0])]
    assert generate(d, [2, 2], 1) == [4]
    with pytest.raises(ValueError):
        q.submit([], 1)

    class Broken(FakeDecoder):
        def decode_greedy(self, s, n):
            raise RuntimeError("x")

    d = Broken()
    q = RequestQueue(d)
    q.submit([1], 1)
    with pytest.raises(RuntimeError):
        q.run()
    assert d.free == 1  # the place is given back


def test_trace_replay_writes_what_is_wanted(tmp_path):
    from cut_b200.trace import replay

    d, said = FakeDecoder(), []
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [4], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [9], "want": [0]}], "end": ["b"]}]
    replay(d, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n\n"), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and d.free == 1
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [6, -6, 1, -1]
    assert not (tmp_path / "1.f32").exists() and np.fromfile(tmp_path / "2.f32", "<f4").tolist() == [9, -9]


@pytest.mark.parametrize("name,struct", [("cutb_dense_desc", L.DenseDesc), ("cutb_residual_norm_desc", L.ResidualNormDesc),
                                         ("cutb_embed_desc", L.EmbedDesc), ("cutb_window_attn_desc", L.WindowAttnDesc)])
def test_descriptor_fields_follow_the_header(name, struct):
    text = open(os.path.join(ROOT, "include", "cutb.h")).read()
    body = re.search(r"typedef struct %s \{(.*?)\} %s;" % (name, name), text, re.S).group(1)
    fields = []
    for decl in re.sub(r"/\*.*?\*/", "", body, flags=re.S).split(";"):
        names = [n.strip().lstrip("*") for n in decl.strip().split(",")]
        if names != [""]:
            fields += [names[0].split()[-1].lstrip("*")] + names[1:]
    assert fields == [f[0] for f in struct._fields_]


def test_argument_validation_needs_no_device():
    lib = L.lib()
    d = L.DenseDesc()
    assert lib.cutb_dense_matmul(C.byref(d), None) == L.ERR_INVALID and b"empty shape" in lib.cutb_last_error()
    d.M, d.K, d.N, d.A, d.lda, d.W, d.ldw, d.C, d.ldc, d.variant = 1, 24, 5, 256, 24, 256, 20, 256, 8, L.DENSE_AUTO
    assert lib.cutb_dense_matmul(C.byref(d), None) == L.ERR_INVALID and b"weight rows" in lib.cutb_last_error()
    d.ldw = 24
    assert lib.cutb_dense_select_variant(C.byref(d)) == L.DENSE_MATVEC
    d.M = 4
    assert lib.cutb_dense_select_variant(C.byref(d)) == L.DENSE_SIMT
    d.a_dtype = L.BF16
    assert lib.cutb_dense_select_variant(C.byref(d)) == L.DENSE_TC
    d.norm_w = 256
    assert lib.cutb_dense_matmul(C.byref(d), None) == L.ERR_INVALID and b"staged norm" in lib.cutb_last_error()
    a = L.WindowAttnDesc()
    for f, v in dict(kv_dtype=L.BF16, out_dtype=L.F32, n_heads=4, n_kv_heads=2, dim=10, vdim=8, k_head=16, v_head=8, ring_rows=64, window=40,
                     rot_dims=4, max_pos=500, q=256, k=256, v=256, k_cache=256, v_cache=256, out=256, n_tokens=30, cos_table=256,
                     sin_table=256).items():
        setattr(a, f, v)
    assert lib.cutb_window_attention(C.byref(a), None) == L.ERR_INVALID and b"do not hold a window" in lib.cutb_last_error()
    a.ring_rows = 100
    assert lib.cutb_window_attention(C.byref(a), None) == L.ERR_INVALID and b"multiple of 64" in lib.cutb_last_error()
    a.ring_rows, a.n_heads = 128, 3
    assert lib.cutb_window_kv_write(C.byref(a), None) == L.ERR_INVALID
    a.n_heads = 4
    assert lib.cutb_window_attention_decode(C.byref(a), None) == L.ERR_INVALID and b"one token" in lib.cutb_last_error()
    n = L.ResidualNormDesc()
    assert lib.cutb_residual_norm(C.byref(n), None) == L.ERR_INVALID
    assert lib.cutb_mingru_scan(None, 0, 4, None, None, L.F32, 4, 1, None) == L.ERR_INVALID
    assert lib.cutb_sequence_advance(None, None, 1, None, None) == L.ERR_INVALID
    assert lib.cutb_embedding_bigram(C.byref(L.EmbedDesc()), None) == L.ERR_INVALID


def test_decoder_needs_a_device():
    if torch.cuda.is_available():
        pytest.skip("a device is present")
    c = bigerax.parse_config(CONFIGS["one"])
    t = torch_weights(random_weights(CONFIGS["one"], 1))
    with pytest.raises(RuntimeError, match="no CPU path"):
        LayerListDecoder(c, bigerax.gather_weights(c, t.__getitem__, t.__contains__))


def test_window_config_helper_defaults():
    assert attention(2, 1, 8, 8, 5)["mixer"]["rot"]["dims"] == 8

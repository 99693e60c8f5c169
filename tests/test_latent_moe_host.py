"""CPU checks of the latent-attention / mixture-of-experts models' host side: configuration and registry, weight layout, argument
validation of the C ABI, and the oracle against itself (absorbed and expanded forms, portions, shared latents)."""
import ctypes as C
import json
import os

import numpy as np
import pytest
import torch

from cut_b200 import _lib as L
from cut_b200 import lenesun, models, ops
from cut_b200.layer_list import LatentAttention, LayerListDecoder, Linear, MixtureOfExperts
from oracle import latent_ref as R
from tests.layer_list_util import row_errors
from tests.lenesun_util import CONFIGS, config, layer, random_weights, safe_tokens, save_model, torch_weights


def test_configuration_reads_every_size_and_constant():
    c = lenesun.parse_config(CONFIGS["mixed"])
    assert (c.width, c.vocab, c.norm_eps, c.residual_mult, c.embed_scale, len(c.layers)) == (136, 211, 1e-5, 0.4, 2.5, 4)
    assert c.parallel and c.norm_center and c.tied_head and c.norm_groups == 1 and c.bigram is None
    a, f = c.layers[2].mixer, c.layers[2].mlp
    assert isinstance(a, LatentAttention) and (a.heads, a.dim, a.rot.dims, a.vdim, a.q_rank, a.kv_rank, a.kv_from) == (2, 40, 16, 16, 24, 48, 0)
    assert a.sink and a.scale == 56 ** -0.5 and a.kv_rows == 0 and c.layers[0].mixer.kv_rows == 64 and c.layers[0].mixer.cache_row == 64
    assert f == MixtureOfExperts(9, 3, 24, 0.7, 1.702, 1.0)
    assert c.layers[1].mlp is None and c.layers[1].mixer.rot.base == 500.0 and c.layers[1].mixer.kv_from is None
    one = lenesun.parse_config(config(24, 9, [{k: v for k, v in layer(1, 2, 2, 2, 3, 4).items() if k != "mlp"}]))  # no mlp entry at all
    assert one.layers[0].mlp is None


@pytest.mark.parametrize("change,what", [
    (lambda c: c["layers"][0].update(type="mystery"), "unknown mixer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="mystery"), "unknown feed-forward"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), "turns as a whole"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=15, rot={"base": 10.0, "dims": 15}), "must be even"),
    (lambda c: c["layers"][0]["mixer"].update(heads=0), "empty latent attention"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "experts per token"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(ff=0), "empty feed-forward"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier layer"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "latents of its own"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "same rank and rotation"),
    (lambda c: c.update(layers=[]), "must not be empty"),
])
def test_configurations_that_make_no_sense_are_refused(change, what):
    c = json.loads(json.dumps(CONFIGS["mixed"]))
    change(c)
    with pytest.raises(ValueError, match=what):
        lenesun.parse_config(c)


def test_registry_chooses_the_class_by_architecture(tmp_path):
    folder = save_model(tmp_path / "m", CONFIGS["odd"], random_weights(CONFIGS["odd"], 1))
    entry, cfg = models.read_config(folder)
    assert entry is models.REGISTRY["Lenesun"] and entry.decoder is LayerListDecoder and cfg == lenesun.parse_config(CONFIGS["odd"])
    assert entry.dtypes == ("bfloat16", "float32")
    assert os.path.exists(os.path.join(folder, "model.safetensors"))


def test_gathered_weights_cover_the_file_and_stack_the_experts():
    cfg, w = CONFIGS["mixed"], random_weights(CONFIGS["mixed"], 2)
    t, asked = torch_weights(w), set()

    def get(n):
        asked.add(n)
        return t[n]

    g = lenesun.gather_weights(lenesun.parse_config(cfg), get, t.__contains__)
    assert asked == set(t)
    assert g["layers"][0]["mlp"]["gate"].shape == (6, 40, 136) and g["layers"][0]["mlp"]["down"].shape == (6, 136, 40)
    assert torch.equal(g["layers"][2]["mlp"]["up"][7], t["l2.mlp.e7.up"]) and "dkv" not in g["layers"][2]["mix"] and "mlp" not in g["layers"][1]


def test_rows_of_a_stacked_matrix_share_its_memory():
    a = Linear([torch.ones(3, 5), 2 * torch.ones(4, 5)], [None, torch.arange(4.0)], "cpu")
    b = a.rows(3, 4)
    assert (b.N, b.K, b.ldw) == (4, 5, 8) and b.w.data_ptr() == a.w[3].data_ptr() and bool((b.w[:, :5] == 2).all()) and b.bias.tolist() == [0, 1, 2, 3]


# ---- the oracle against itself ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", list(CONFIGS))
def test_oracle_portions_and_token_by_token(name):
    cfg = CONFIGS[name]
    ref = R.LatentReference(cfg, random_weights(cfg, 3))
    toks = safe_tokens(ref, 40, 1, 1e-3)
    whole = ref.run(toks)
    for cuts in ([0, 2, 4, 25, 40], list(range(41))):
        ref.reset()
        assert row_errors(np.concatenate([ref.run(toks[a:b]) for a, b in zip(cuts, cuts[1:])]), whole).max() < 1e-10


def test_absorbed_scores_and_values_equal_the_expanded_ones():
    rng = np.random.default_rng(0)
    H, dim, rot, vdim, rank, n = 3, 5, 4, 6, 7, 9
    c, r, uk, uv = (rng.standard_normal(s) for s in ((n, rank), (n, rot), (H * dim, rank), (H * vdim, rank)))
    q, sink = rng.standard_normal((n, H, dim + rot)), rng.standard_normal(H)
    k, v = R.latent_keys_values(c, r, uk, uv, H)
    want = R.sink_attention(q, k, v, 0, 0.4, sink)
    qa = np.einsum("thd,hdr->thr", q[:, :, :dim], uk.reshape(H, dim, rank))
    row = np.concatenate([c, r], axis=1)[:, None, :].repeat(H, 1)
    lat = R.sink_attention(np.concatenate([qa, q[:, :, dim:]], axis=2), row, c[:, None, :].repeat(H, 1), 0, 0.4, sink).reshape(n, H, rank)
    assert np.allclose(np.einsum("thr,hvr->thv", lat, uv.reshape(H, vdim, rank)).reshape(n, -1), want)


def test_oracle_sinks_clamps_norms_and_choices():
    assert np.allclose(R.layer_norm(np.array([[1.0, 3.0]]), np.array([2.0, 1.0]), 0.0), [[-2.0, 1.0]])
    assert np.allclose(R.rms_norm(np.array([[3.0, 4.0]]), np.ones(2), 0.0), np.array([[3.0, 4.0]]) / np.sqrt(12.5))
    one = np.ones((1, 1, 1))
    assert np.allclose(R.sink_attention(one, one, one, 0, 0.0, np.array([np.log(3.0)])), 0.25) and R.sink_attention(one, one, one, 0, 0.0, None) == 1.0
    assert np.allclose(R.clamped_glu(np.array([9.0, -9.0]), np.array([9.0, -9.0]), 2.0), [2 * R.sigmoid(3.404) * 3, -9 * R.sigmoid(-1.702 * 9) * -1])
    ids, w = R.choose_experts(np.array([1.0, 4.0, 1.0, 3.0]), 2)
    assert ids.tolist() == [1, 3] and np.allclose(w, [np.e / (np.e + 1), 1 / (np.e + 1)])
    x = R.turn_pairs(np.array([[1.0, 0.0, 0.0, 1.0]]), [2], 100.0)
    assert np.allclose(x, [[np.cos(2), np.sin(2), -np.sin(0.2), np.cos(0.2)]])


# ---- argument validation (nothing is launched: no GPU here) ------------------------------------------------------------------
def _refused(name, d, status=L.ERR_INVALID):
    assert getattr(L.lib(), name)(C.byref(d), None) == status, name
    assert L.lib().cutb_last_error().decode()


def test_latent_arguments_are_checked():
    cache, q = torch.zeros(64, 64), torch.zeros(4, 400)
    tab = torch.zeros(64, 4)
    def make(T=1, **k):
        return ops.latent_desc(cache, 2, 16, 8, 16, 40, scale=1.0, eps=1e-5, max_pos=64, n_tokens=T, cos_t=tab, sin_t=tab, **k)
    n = ops.latent_workspace_bytes(make())
    assert n > 0 and L.lib().cutb_latent_splits(C.byref(make())) >= 1 and L.lib().cutb_latent_splits(C.byref(make(T=3))) == 1
    assert ops.latent_workspace_bytes(make(T=3)) == 0
    _refused("cutb_latent_kv_write", make())                                  # nothing to do
    _refused("cutb_latent_attention", make(q=q, qa=q), L.ERR_WORKSPACE)
    _refused("cutb_latent_attention", make(T=2, q=q, qa=q))                   # no output
    _refused("cutb_latent_attention", make(T=2, q=q, qa=q, out=q, lat=q, lat_norm_w=q))
    _refused("cutb_latent_values", make(out=q))
    for field, value in (("rank", 2000), ("rot_dim", 7), ("rot_at", 36), ("ld_cache", 44), ("n_heads", 0), ("max_pos", 0), ("cos_table", None)):
        d = make(T=2, q=q, qa=q, out=q)
        setattr(d, field, value)
        _refused("cutb_latent_attention", d)
    d = make(T=2, q=q, k_exp=q, v_exp=q, out=q)
    assert not L.lib().cutb_latent_prefill_supported(C.byref(d))               # (an fp32 cache)
    _refused("cutb_latent_prefill", d, L.ERR_UNSUPPORTED)
    d.kv_dtype = L.BF16
    assert L.lib().cutb_latent_prefill_supported(C.byref(d))
    for field, value in (("dim", 12), ("rot_dim", 248), ("vdim", 264)):
        e = make(T=2, q=q, k_exp=q, v_exp=q, out=q)
        e.kv_dtype = L.BF16
        setattr(e, field, value)
        assert not L.lib().cutb_latent_prefill_supported(C.byref(e)), field


def test_mixture_arguments_are_checked():
    x, i = torch.zeros(16, 64), torch.zeros(16, 4, dtype=torch.int32)
    w = torch.zeros(4 * 16, 64, dtype=torch.bfloat16)
    route = lambda E, top: ops.moe_route_desc(x, E, top, x, i, i, i)
    for E, top in ((4, 5), (4, 0), (2000, 4), (80, 4)):
        _refused("cutb_moe_route", route(E, top))
    mm = lambda **k: ops.moe_matmul_desc(x, w, 64, i, 4, 16, 1, x, **k)
    _refused("cutb_moe_matmul", mm(variant=L.DENSE_TC), L.ERR_UNSUPPORTED)     # fp32 rows
    _refused("cutb_moe_matmul", mm(variant=L.DENSE_MATVEC))
    _refused("cutb_moe_matmul", mm(glu=7))
    d = mm()
    d.ldw = 60
    _refused("cutb_moe_matmul", d)
    d = ops.moe_scatter_desc(x, 64, i, 4, x.to(torch.bfloat16))
    _refused("cutb_moe_scatter", d)                                           # another element type
    ex = lambda **k: ops.expert_desc(4, k.pop("top", 2), 64, 8, w, i, x, **k)
    _refused("cutb_expert_up", ex(x=x))                                       # no logits
    _refused("cutb_expert_up", ex(logits=x, x=x, top=5))
    _refused("cutb_expert_up", ex(logits=x, x=x, dense=w, dense_K=64, xd=x))  # the dense matrix has no output
    _refused("cutb_expert_down", ex())
    _refused("cutb_expert_down", ex(dense=w[:32], dense_K=64, xd=x, out=x))   # not width rows
    d = ops.expert_desc(400, 65, 64, 8, w, i, x, logits=x, x=x)
    _refused("cutb_expert_up", d, L.ERR_UNSUPPORTED)


def test_batched_products_and_parts_are_checked():
    a, w, out = torch.zeros(4, 96), torch.zeros(3 * 8, 32, dtype=torch.bfloat16), torch.zeros(4, 24)
    good = ops.batch_desc(a, w, 32, out, 3, 32, 8)
    assert L.lib().cutb_dense_select_variant(C.byref(good)) == L.DENSE_SIMT
    assert L.lib().cutb_dense_select_variant(C.byref(ops.batch_desc(a[:1], w, 32, out, 3, 32, 8))) == L.DENSE_MATVEC
    for change in (dict(a_batch=40), dict(c_batch=9), dict(unary_op=133), dict(bias=a.data_ptr())):
        d = ops.batch_desc(a, w, 32, out, 3, 32, 8)
        for k, v in change.items():
            setattr(d, k, v)
        _refused("cutb_dense_matmul", d)
    d = L.ResidualNormDesc()
    d.x = d.pre_w = d.h = a.data_ptr()
    d.ldx = d.ldh = 96
    d.rows, d.dim, d.groups, d.n_parts = 4, 96, 1, 2
    _refused("cutb_residual_norm", d)                                         # parts without rows

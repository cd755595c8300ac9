"""Layer-stack models without a GPU: configuration reader, weight names, registry, cache layout, ragged batches, the bias
buckets, and the oracle's own consistency (its closed forms against its recurrences)."""
import json
import math

import pytest
import torch

from tests import roluzen_oracle as O
from tests import stack_cases as C
from tests import tovalix_oracle as TO
from tests import zigipel_oracle as ZG
from tests import zikezen_oracle as ZO


@pytest.mark.parametrize("name", sorted(C.CASES))
def test_checkpoint_round_trip(tmp_path, name):
    from safetensors.torch import load_file
    from tunix_b200.models.automodel import AutoModel
    from tunix_b200.models.safetensors_saver import save_lora_merged_model_as_safetensors
    from tunix_b200.models.stack import StackModel
    cfg = C.CASES[name]
    src = C.write(tmp_path / (cfg["architecture"].lower() + "-tiny"), cfg, C.weights(cfg))      # a directory name that could be taken for a preset
    model, path = AutoModel.from_pretrained(src, model_source="local")
    assert isinstance(model, StackModel) and path == src
    assert model.config.runs() == O.layer_runs(cfg) and model.config.norm_eps == cfg["norm"]["eps"]
    save_lora_merged_model_as_safetensors(model, str(tmp_path / "out"), source_dir=src)
    a, b = load_file(src + "/model.safetensors"), load_file(str(tmp_path / "out" / "model.safetensors"))
    assert a.keys() == b.keys() and all(torch.equal(a[k], b[k]) for k in a)
    again, _ = AutoModel.from_pretrained("anything", model_source="local", model_path=str(tmp_path / "out"), dtype=torch.float32)
    assert again.embed_tokens.dtype == torch.float32


def test_constants_come_from_config_json(tmp_path):
    from tunix_b200.models.hf_config import config_from_hf
    cfg = C.CASES["mixed"]
    src = C.write(tmp_path / "m", cfg, C.weights(cfg, buckets=14))
    c = config_from_hf(src)
    left, right = c.layer_specs[1].mixer.left, c.layer_specs[1].mixer.right
    want = cfg["layers"][1]["mixer"]
    assert (left.scale, left.bias_max, left.window, left.keep_first) == (want["left"]["scale"], 40, 20, 3)
    assert left.buckets == 14                                          # told by the tensor's shape only
    assert (right.gate_cap, right.dim, right.vdim) == (9.0, 24, 40)
    assert c.layer_specs[2].ff is None and c.layer_specs[3].mixer.conv == 2 and c.streams == 3 and c.loop == (1, 3, 2)
    with pytest.raises(ValueError, match="mixer"):
        config_from_hf(dict(cfg, layers=[dict(cfg["layers"][0], type="other")]))
    with pytest.raises(ValueError, match="feed-forward"):
        config_from_hf(dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "sparse", "ff": 8})]))


def test_cache_layout_is_per_pass():
    from tunix_b200.models.hf_config import config_from_hf
    c = config_from_hf(C.CASES["mixed"])
    assert c.runs() == [0, 1, 2, 1, 2, 3]
    assert c.kv_rows() == [None, (32, 48), (32, 48), (32, 48), (32, 48), None]
    states = c.state_shapes()
    assert states[0] == {"s": (80,), "ring": (4, 80)} and states[5] == {"s": (80,), "ring": (2, 80)}
    assert states[1] == {"S": (2, 24, 40), "n": (2, 2, 24), "m": (2, 2)}


def test_tovalix_constants_come_from_config_json(tmp_path):
    from tunix_b200.models.hf_config import config_from_hf
    cfg = C.CASES["shared"]
    src = C.write(tmp_path / "m", cfg, C.tovalix_weights(cfg, rank=5))
    c = config_from_hf(src)
    assert (c.norm_groups, c.token_side, c.embed_norm, c.norm_eps, c.streams, c.loop) == (3, 8, True, 1e-5, 0, None)
    a, b = c.layer_specs[1].mixer, c.layer_specs[3].mixer
    assert (a.scale, a.softcap, a.chunk, a.rot_dims, a.rot_base, a.kv_from) == (0.6, 6.0, 20, 8, 900.0, None)
    assert (b.heads, b.chunk, b.softcap, b.kv_from) == (2, 33, 3.0, 1)
    assert c.layer_specs[0].mixer.decay_rank == 5                      # told by the tensor's shape only
    assert [s.ff for s in c.layer_specs] == [56, 64, None, None, 56] and c.layer_specs[0].ff_kind == "xielu"
    assert (c.num_heads, c.num_kv_heads, c.head_dim) == (4, 2, 16)
    with pytest.raises(ValueError, match="mixer"):                     # a design has its own layer types only
        config_from_hf(dict(cfg, layers=[C.rglru()]))
    for layers in ([C.rotary(kv_from=1), C.rotary()], [C.wkv(), C.rotary(kv_from=0)], [C.rotary(), C.rotary(kv_from=0), C.rotary(kv_from=1)],
                   [C.rotary(), C.rotary(kv_heads=4, kv_from=0)]):
        with pytest.raises(ValueError, match="keys and values"):
            config_from_hf(dict(cfg, layers=layers))
    with pytest.raises(ValueError, match="groups"):
        config_from_hf(dict(cfg, norm={"eps": 1e-5, "groups": 5}))


def test_shared_keys_take_no_pages():
    from tunix_b200.generate.engine import PagePool
    from tunix_b200.models.hf_config import config_from_hf
    c = config_from_hf(C.CASES["shared"])
    assert c.kv_rows() == [None, (32, 48), None, None, None] and c.kv_sources() == [0, 1, 2, 1, 4]
    assert c.replace(loop=(0, 2, 2)).kv_sources() == [0, 1, 2, 3, 4, 3, 6]      # the latest pass of the layer
    with pytest.raises(ValueError, match="has not run"):
        c.replace(loop=(0, 2, 0))
    states = c.state_shapes()
    assert states[0] == {"S": (3, 16, 16), "last": (48,)} and states[2] == {"S": (2, 24, 40)} and states[1] == states[3] == {}
    pool = PagePool(c, 4, 16, 2, 4, "cpu", torch.float32, prefix_caching=False)
    assert pool.k[3] is None and pool.v[1].shape == (4, 16, 48)
    assert pool.state.nbytes_per_slot() == 4 * (3 * 256 + 48 + 2 * 960 + 2 * 576 + 48)


def test_pool_and_states_on_cpu():
    from tunix_b200.generate.engine import PagePool
    from tunix_b200.models.hf_config import config_from_hf
    c = config_from_hf(C.CASES["mixed"])
    pool = PagePool(c, 6, 16, 2, 4, "cpu", torch.float32, prefix_caching=False)
    assert pool.k[0] is None and pool.k[1].shape == (6, 16, 32) and pool.v[1].shape == (6, 16, 48)
    assert pool.state[1]["S"].shape == (2, 2, 24, 40) and pool.state[1]["S"].dtype == torch.float32
    assert pool.state.nbytes_per_slot() == 4 * (80 + 320 + 80 + 160 + 4 * (2 * 24 * 40 + 2 * 2 * 24 + 4))
    pool.open(0, [1] * 20, 0)
    pool.grow(0, 60)
    assert len(pool.pages_of(0)) == 4
    with pytest.raises(pool.Error):
        pool.open(1, [1] * 60, 0)
    pool.release(0)
    pool.open(1, [1] * 60, 0)


def test_registry_presets_and_names():
    from tunix_b200.models import naming, registry
    from tunix_b200.models.config import get_config
    from tunix_b200.models.transformer import create_model
    assert registry.get_family("roluzen").family == "roluzen" and registry.family_of_hf_id("x/Roluzen-2B").family == "roluzen"
    assert naming.config_for("roluzen-2b") == get_config("roluzen_2b")
    model = create_model(get_config("roluzen_tiny"), seed=3)
    assert model.config.runs() == [0, 1, 2, 1, 2]
    assert torch.equal(model.layers[0].hc1.mix, torch.eye(3)) and model.layers[1].mixer.right.f_proj.bias.eq(3).all()
    assert registry.get_family("tovalix").family == "tovalix" and naming.config_for("tovalix-8b") == get_config("tovalix_8b")
    assert naming.get_model_family("x/Tovalix-2B") == "tovalix"
    small = create_model(get_config("tovalix_tiny"), seed=3)
    assert small.config.kv_sources() == [0, 1, 2, 3, 4, 2] and small.layers[5].mixer.k_proj is None
    assert small.num_params == get_config("tovalix_tiny").num_params()
    with pytest.raises(ValueError, match="loop"):
        get_config("roluzen_tiny").replace(loop=(2, 5, 1))
    with pytest.raises(NotImplementedError):
        model(torch.zeros(1, 1, dtype=torch.long), cache=[])


@pytest.mark.parametrize("rows,far", [(11, 40), (16, 100), (8, 64), (7, 33), (32, 4096), (6, 12)])
def test_distance_buckets(rows, far):
    from tunix_b200.models.mixers import distance_buckets
    got = distance_buckets(rows, far)
    want = [O.distance_bucket(n, rows, far) for n in range(far + 1)]
    # where the logarithm is an integer in exact arithmetic the two may round apart; nowhere else
    for n, (a, b) in enumerate(zip(got.tolist(), want)):
        if a != b:
            half = rows // 2
            x = math.log(n / half) / math.log(far / half) * (rows - half)
            assert abs(x - round(x)) < 1e-9, n
    assert got[far] == rows - 1 and O.distance_bucket(10 * far, rows, far) == rows - 1


def test_ragged_batch_layout():
    from tunix_b200.ops.ragged import RaggedBatch
    rb = RaggedBatch.build([(3, 0, [5, 6, 7]), (1, 9, [8]), (0, 2, [1, 2])], "cpu")
    assert rb.tokens.tolist() == [5, 6, 7, 8, 1, 2] and rb.cu.tolist() == [0, 3, 4, 6]
    assert rb.slot.tolist() == [3, 1, 0] and rb.pos0.tolist() == [0, 9, 2] and rb.ent.tolist() == [0, 0, 0, 1, 2, 2]
    assert not rb.decode
    t0, ent, first, n = rb.tiles(2)
    assert t0.tolist() == [0, 2, 3, 4] and ent.tolist() == [0, 0, 1, 2] and first.tolist() == [0, 2, 3] and n == 4
    assert RaggedBatch.build([(0, 4, [1]), (2, 7, [3])], "cpu").decode


def test_joint_weights_share_memory_and_follow_updates():
    from tunix_b200.models.config import get_config
    from tunix_b200.models.stack_exec import StackExecutor
    from tunix_b200.models.transformer import create_model
    model = create_model(get_config("roluzen_tiny"), seed=0)
    ex = StackExecutor(model)
    before = {k: v.data_ptr() for k, v in ex.w[1].items() if v is not None}
    left = model.layers[1].mixer.left
    n = left.q_proj.weight.shape[0]
    assert left.k_proj.weight.data_ptr() == ex.w[1]["proj"][n:].data_ptr()
    with torch.no_grad():
        left.k_proj.weight.fill_(2.0)
        left.rel.fill_(1.5)
        model.layers[0].mixer.y_proj.bias.fill_(0.25)
    ex.refresh()
    assert {k: v.data_ptr() for k, v in ex.w[1].items() if v is not None} == before
    assert ex.w[1]["proj"][n].eq(2).all() and ex.w[1]["bias"].eq(1.5).all() and ex.w[0]["proj_bias"][0] == 0.25
    model.layers[1].mixer.left.q_proj.lora_a = torch.nn.Parameter(torch.zeros(1, 1))
    with pytest.raises(NotImplementedError, match="adapters"):
        ex.refresh()


def test_joint_weights_of_memories_and_rotary_attention():
    from tunix_b200.models.config import get_config
    from tunix_b200.models.stack_exec import StackExecutor, rope_table
    from tunix_b200.models.transformer import create_model
    model = create_model(get_config("tovalix_tiny"), seed=0)
    ex = StackExecutor(model)
    before = {k: v.data_ptr() for d in ex.w for k, v in d.items() if v is not None}
    with torch.no_grad():
        model.layers[0].mixer.mu_g.fill_(0.125)
        model.layers[2].mixer.v_proj.bias.fill_(3.0)
        model.layers[1].mixer.v_proj.weight.fill_(2.0)
    ex.refresh()
    assert {k: v.data_ptr() for d in ex.w for k, v in d.items() if v is not None} == before
    assert ex.w[0]["mu"][3].eq(0.125).all() and "proj" not in ex.w[0]
    assert ex.w[2]["proj_bias"][-1] == 3.0 and ex.w[1]["proj"][-1].eq(2).all() and ex.w[1]["gates_bias"] is None
    assert ex.w[5]["proj"].shape[0] == 4 * 32                           # queries only
    cos, sin = rope_table(3000, 6, 900.0, "cpu")
    a = 2999 * 900.0 ** (-4 / 6)
    assert cos[0].eq(1).all() and abs(cos[2999, 2].item() - math.cos(a)) < 1e-7 and abs(sin[2999, 2].item() - math.sin(a)) < 1e-7


def test_oracle_recurrences_against_their_unrolled_sums():
    """The token-by-token memories of the second oracle against direct sums over all earlier tokens."""
    torch.manual_seed(1)
    T, H, d, dv = 20, 2, 5, 4
    q, k, v = (torch.randn(T, H, n, dtype=torch.float64) for n in (d, d, dv))
    f, u = torch.rand(T, H, d, dtype=torch.float64), torch.randn(H, d, dtype=torch.float64)
    wkv, hgrn = TO.wkv_recurrence(q, k, v, f, u), TO.hgrn2_recurrence(q, f, v)
    for t in range(T):
        a, b = torch.zeros(H, dv).double(), torch.zeros(H, dv).double()
        for s in range(t + 1):
            after = f[s + 1:t].prod(0) if s < t else u                  # decays between the two tokens, or the bonus
            a += (q[t] * after * k[s]).sum(-1, keepdim=True) * v[s]
            b += (q[t] * f[s + 1:t + 1].prod(0) * (1 - f[s])).sum(-1, keepdim=True) * v[s]
        assert torch.allclose(wkv[t], a) and torch.allclose(hgrn[t], b)


def test_oracle_details():
    x = torch.tensor([[3.0, 4.0, 0.0, 2.0]], dtype=torch.float64)
    got = TO.group_norm(x, torch.tensor([1.0, 1.0, 1.0, 2.0]).double(), 2, 0.0)
    assert torch.allclose(got, torch.tensor([[3 / 12.5 ** 0.5, 4 / 12.5 ** 0.5, 0.0, 2 * 2 ** 0.5]]).double())
    z, p, q = torch.tensor([-1.0, 0.0, 2.0]).double(), torch.tensor(0.3).double(), torch.tensor(-0.7).double()
    sp = lambda a: math.log(1 + math.exp(a))  # noqa: E731
    want = [(0.5 + sp(-0.7)) * (math.exp(-1) - 1 + 1) - 0.5, 0.0, sp(0.3) * 4 + 1]
    assert torch.allclose(TO.xielu(z, p, q), torch.tensor(want).double())
    assert TO.visible(19, 0, 20) and not TO.visible(20, 19, 20) and not TO.visible(20, 21, 20)
    h = torch.randn(5, 3).double()
    assert torch.equal(TO.token_shift(h, torch.ones(3).double())[1:], h[:-1]) and TO.token_shift(h, torch.ones(3).double())[0].eq(0).all()


def test_oracle_memory_against_its_unrolled_sum():
    """The token-by-token matrix memory of the oracle against the direct sum over all earlier tokens."""
    torch.manual_seed(0)
    T, m = 30, {"heads": 2, "dim": 6, "vdim": 5, "gate_cap": 7.0}
    D = 16
    w = {n: torch.randn(r, D, dtype=torch.float64) for n, r in (("q", 12), ("k", 12), ("v", 10), ("g", 10), ("i", 2), ("f", 2))}
    w.update({"i.b": torch.randn(2).double(), "f.b": torch.randn(2).double() + 2, "norm": torch.ones(10).double(),
              "o": torch.eye(10).double()})
    h = torch.randn(T, D, dtype=torch.float64)
    got = O.matrix_memory(w, "", h, m, 1e-6)
    ig = 7 * torch.tanh((h @ w["i"].T + w["i.b"]) / 7)
    F = torch.nn.functional.logsigmoid(7 * torch.tanh((h @ w["f"].T + w["f.b"]) / 7)).cumsum(0)
    q, k, v = (h @ w["q"].T).view(T, 2, 6) / 6 ** 0.5, (h @ w["k"].T).view(T, 2, 6), (h @ w["v"].T).view(T, 2, 5)
    out = torch.zeros(T, 2, 5, dtype=torch.float64)
    for t in range(T):
        for a in range(2):
            lw = F[t, a] - F[:t + 1, a] + ig[:t + 1, a]
            top = max(F[t, a].item(), lw.max().item())
            s = torch.exp(lw - top) * (k[:t + 1, a] @ q[t, a])
            out[t, a] = s @ v[:t + 1, a] / (max(abs(s.sum().item()), math.exp(-top)) + 1e-6)
    want = O.rms(out, 1e-6).reshape(T, 10) * torch.sigmoid(h @ w["g"].T)
    assert torch.allclose(got, want, atol=1e-9)


def test_trace_runner_help_names_its_options():
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    path = os.path.join(root, "bin", "trace_run")
    assert os.access(path, os.X_OK)
    out = subprocess.run([sys.executable, path, "--help"], capture_output=True, text=True).stdout
    assert all(o in out for o in ("--model", "--dtype", "--out", "--max-tokens"))


def test_configs_are_json():
    for cfg in C.CASES.values():
        assert json.loads(json.dumps(cfg)) == cfg


# ------------------------------------------------------------------------------------------------ Zikezen
def test_zikezen_constants_come_from_config_json(tmp_path):
    from tunix_b200.models.hf_config import config_from_hf
    cfg = C.CASES["looped"]
    src = C.write(tmp_path / "m", cfg, C.zikezen_weights(cfg, rank=7))
    c = config_from_hf(src)
    assert (c.family, c.embed_factor, c.positions, c.max_position, c.final_logit_softcap, c.token_side) == ("zikezen", 1.7, 512, 512, 12.0, 8)
    assert c.post_norms and c.loop_embed and c.loop == (0, 3, 3) and c.streams == 0 and not c.is_moe
    m = c.layer_specs[1].mixer
    assert (m.left_scale, m.right_scale, m.right.tau, m.right.decay_rank) == (1.1, 0.4, 12.0, 7)
    a = m.left
    assert (a.heads, a.kv_heads, a.window, a.scale, a.rot_dims, a.rot_base, a.rot_scaling) == (2, 2, 7, 0.4, 8, 700.0, (5.0, 1.0, 3.5, 60.0))
    assert a.interleaved and a.head_weights and a.sink == 0.0 and not a.out_bias and a.softcap == 0.0 and a.chunk == 0
    assert [(s.ff, s.ff_kind, s.experts, s.top) for s in c.layer_specs] == [(40, "experts", 6, 2), (None, "glu", 0, 0), (56, "experts", 5, 5),
                                                                            (72, "glu", 0, 0)]
    assert c.runs() == [0, 1, 2] * 3 + [3] and c.restarts() == {3, 6}
    assert config_from_hf(C.CASES["ragged"]).restarts() == {2} and config_from_hf(C.CASES["ragged"]).layer_specs[0].mixer.left.rot_scaling is None
    plain = config_from_hf(dict(cfg, loop=None, logit_softcap=None))
    assert plain.restarts() == set() and plain.final_logit_softcap == 0.0
    with pytest.raises(ValueError, match="mixer"):
        config_from_hf(dict(cfg, layers=[C.hgrn2()]))
    with pytest.raises(ValueError, match="feed-forward"):               # only designs that have experts take them
        config_from_hf(dict(C.CASES["shared"], layers=[dict(C.wkv(), mlp=cfg["layers"][0]["mlp"])]))
    with pytest.raises(ValueError, match="experts"):
        config_from_hf(dict(cfg, loop=None, layers=[C.beside(experts=(3, 4))]))


def test_stored_heads_and_cache_rows():
    from tunix_b200.models.hf_config import config_from_hf
    c = config_from_hf(C.CASES["blocks"])
    specs = [s.mixer.left for s in c.layer_specs]
    assert [a.stored(torch.bfloat16) for a in specs] == [(64, 64), (128, 128), (128, 128)]
    assert [a.stored(torch.float32) for a in specs] == [(40, 56), (96, 80), (128, 128)]
    assert c.kv_rows() == [(192, 192), (128, 128), (256, 256), (128, 128), (256, 256)]
    assert c.kv_rows(torch.float32)[:2] == [(120, 168), (96, 80)]
    assert config_from_hf(C.CASES["ragged"]).kv_rows() == [(10, 6), (18, 42), (18, 42), (32, 48)]
    assert c.state_shapes()[0] == {"S": (2, 40, 72)} and len(c.state_shapes()) == 5


def test_zikezen_presets_and_parameters():
    from tunix_b200.models import naming, registry
    from tunix_b200.models.config import get_config
    from tunix_b200.models.transformer import create_model
    assert registry.get_family("zikezen").family == "zikezen" and registry.family_of_hf_id("x/Zikezen-2B").family == "zikezen"
    assert naming.config_for("zikezen-8b") == get_config("zikezen_8b") and naming.get_model_family("x/Zikezen-2B") == "zikezen"
    model = create_model(get_config("zikezen_tiny"), seed=3)
    assert model.num_params == get_config("zikezen_tiny").num_params() and model.config.runs() == [0, 1, 2, 1, 2, 3]
    assert model.layers[0].post_attn_norm.weight.eq(1).all() and model.layers[1].mlp.correction.eq(0).all()
    assert model.layers[0].mixer.right.a2_proj.bias.eq(2).all() and model.layers[1].mlp.gate_proj.std() > 0.01
    with pytest.raises(ValueError, match="position"):
        model(torch.zeros(1, 513, dtype=torch.long))


def test_missing_experts_are_named(tmp_path):
    from safetensors.torch import load_file, save_file
    from tunix_b200.models.automodel import AutoModel
    cfg = C.CASES["looped"]
    src = C.write(tmp_path / "m", cfg, C.weights(cfg))
    t = load_file(src + "/model.safetensors")
    del t["l0.mlp.e3.up"]
    save_file(t, src + "/model.safetensors")
    with pytest.raises(KeyError, match="up_proj#3"):
        AutoModel.from_pretrained(src, model_source="local")


def test_parameters_joined_side_by_side_follow_updates():
    from tunix_b200.models.config import get_config
    from tunix_b200.models.stack_exec import StackExecutor
    from tunix_b200.models.transformer import create_model
    model = create_model(get_config("zikezen_tiny"), seed=0)
    ex = StackExecutor(model)
    before = {(i, k): v.data_ptr() for i, d in enumerate(ex.w) for k, v in d.items() if v is not None}
    mix, mlp = model.layers[1].mixer, model.layers[1].mlp
    want = torch.cat([mix.left.o_proj.weight, mix.right.o_proj.weight], 1)
    with torch.no_grad():
        mix.right.o_proj.weight.mul_(2.0)
        mlp.up_proj[3].fill_(0.5)
        mix.left.v_proj.bias.fill_(3.0)
    ex.refresh()
    assert {(i, k): v.data_ptr() for i, d in enumerate(ex.w) for k, v in d.items() if v is not None} == before
    n = mix.left.o_proj.weight.shape[1]
    assert torch.equal(ex.w[1]["o"][:, :n], want[:, :n]) and torch.equal(ex.w[1]["o"][:, n:], 2 * want[:, n:])
    gu, F = ex.w[1]["experts_gu"], mlp.gate_proj.shape[1]
    assert gu.is_contiguous() and torch.equal(gu[:, :F], mlp.gate_proj) and gu[3, F:].eq(0.5).all() and "experts_gu" not in ex.w[0]
    a = mix.spec.left
    q, kv = a.heads * a.dim, a.kv_heads * (a.dim + a.vdim)
    b = ex.w[1]["proj_bias"]
    assert b[q + a.kv_heads * a.dim:q + kv].eq(3).all() and b[q + kv:].eq(0).all() and b.numel() == ex.w[1]["proj"].shape[0]
    assert set(ex.pack_sources()[1]) == {"proj", "o"} and "down" in ex.pack_sources()[0]


@pytest.mark.parametrize("scaling", [None, (5.0, 1.0, 3.5, 60.0), (8.0, 1.0, 4.0, 8192.0), (3.0, 2.0, 2.0, 500.0), (1.0, 1.0, 4.0, 100.0)])
def test_rope_frequencies(scaling):
    from tunix_b200.models.stack_exec import rope_frequencies
    for dims, base in ((32, 5e5), (8, 700.0), (2, 40.0), (0, 1.0)):
        rot = {"dims": dims, "base": base}
        if scaling:
            rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
            rot["scaling"]["high"] += 1e-9 * (scaling[1] == scaling[2])        # the oracle divides by the band's width
        assert torch.allclose(rope_frequencies(dims, base, scaling), ZO.frequencies(rot), rtol=1e-6)


def test_zikezen_oracle_details():
    s = torch.tensor([0.0, math.log(2.0), -math.inf]).double()
    assert torch.allclose(ZO.sink_softmax(s), torch.tensor([0.25, 0.5, 0.0]).double())
    assert torch.allclose(ZO.sink_softmax(s + 300), torch.tensor([1 / 3, 2 / 3, 0.0]).double()) and ZO.sink_softmax(s - 300).sum() < 1e-100
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0]]]).double()
    got = ZO.rotate(x, torch.tensor([3]), {"dims": 4, "base": 100.0})[0, 0]
    a, b = 3.0, 0.3
    assert torch.allclose(got, torch.tensor([math.cos(a), math.sin(a), -2 * math.sin(b), 2 * math.cos(b), 5.0]).double())
    f = ZO.frequencies({"dims": 6, "base": 1000.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100}})
    turns = [100 / (2 * math.pi) * 1000.0 ** (-i / 3) for i in range(3)]                 # 15.9, 1.59, 0.159
    mid = (turns[1] - 1) / 3
    assert torch.allclose(f, torch.tensor([1.0, 0.1 * (mid + (1 - mid) / 4), 0.01 / 4]).double())
    r = ZO.route(torch.tensor([[0.0, 1.0, 2.0]]).double(), torch.eye(3).double(), torch.tensor([0.9, 0.0, 0.0]).double(), 2)
    p = torch.softmax(torch.tensor([0.0, 1.0, 2.0]).double(), 0)
    assert torch.allclose(r[0], torch.stack([p[0], p[1] * 0, p[2]]))
    assert torch.allclose(ZO.decays(torch.tensor([0.0, -800.0]).double(), 4.0), torch.tensor([0.5 ** 0.25, math.exp(-200)]).double())
    assert ZO.visible(19, 0, 20) and not ZO.visible(20, 0, 20) and not ZO.visible(3, 4, 20)
    assert ZO.layer_runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == \
        [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]


def test_zikezen_memory_against_its_unrolled_sum():
    torch.manual_seed(2)
    T, H, d, dv = 12, 2, 4, 3
    q, k, v, a = (torch.randn(T, H, n, dtype=torch.float64) for n in (d, d, dv, d))
    a = torch.sigmoid(a)
    got = ZO.gla_recurrence(q, k, v, a)
    for t in range(T):
        want = sum((q[t] * a[s + 1:t + 1].prod(0) * k[s]).sum(-1, keepdim=True) * v[s] for s in range(t + 1))
        assert torch.allclose(got[t], want)


def test_sequences_stay_within_the_learned_positions():
    from types import SimpleNamespace

    from tunix_b200.generate.engine import check_length
    from tunix_b200.models.hf_config import config_from_hf
    eng = SimpleNamespace(cfg=config_from_hf(C.CASES["looped"]))
    check_length(eng, 512)
    with pytest.raises(ValueError, match="positions"):
        check_length(eng, 513)
    check_length(SimpleNamespace(cfg=config_from_hf(C.CASES["shared"])), 10 ** 6)
    check_length(SimpleNamespace(), 10 ** 6)


# ------------------------------------------------------------------------------------------------ Zigipel
def test_zigipel_constants_come_from_config_json():
    from tunix_b200.models.hf_config import config_from_hf
    from tunix_b200.models.mixers import YarnScaling
    cfg = C.CASES["pairs"]
    c = config_from_hf(cfg)
    assert (c.family, c.bigram, c.logit_scale, c.activation, c.streams, c.token_side) == ("zigipel", (53, 5, 3), 0.4, "gelu", 0, 0)
    assert c.parallel_ff and c.token_shift and c.ff_bias and c.loop_input and not c.loop_embed and not c.post_norms
    assert c.loop == (1, 3, 2) and c.runs() == [0, 1, 2, 1, 2, 3] and c.loop_starts() == {1: 0, 3: 1}
    a, b = c.layer_specs[0].mixer, c.layer_specs[2].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.window, a.keep_first) == (4, 2, 16, 24, 0.6, 20, 3)
    assert (b.heads, b.dim, b.rot_dim, b.vdim, b.kv_rank, b.scale, b.window, b.rot_dims, b.rot_base) == (4, 24, 16, 8, 24, 0.5, 70, 16, 700.0)
    assert b.rot_scaling == YarnScaling(5.0, 60.0, 3.0, 0.5) and [s.ff for s in c.layer_specs] == [56, 40, None, None]
    assert config_from_hf(C.CASES["crooked"]).loop_starts() == {0: 0, 3: 1, 6: 2} and config_from_hf(C.CASES["slabs"]).loop_starts() == {}
    assert config_from_hf(dict(cfg, logit_scale=None, embedding={})).bigram is None
    plain = dict(cfg["layers"][1]["mixer"], rot={"dims": 8, "base": 5.0})
    assert config_from_hf(dict(cfg, loop=None, layers=[dict(cfg["layers"][1], mixer=plain)])).layer_specs[0].mixer.rot_scaling is None
    with pytest.raises(ValueError, match="mixer"):
        config_from_hf(dict(cfg, layers=[C.wkv()]))
    with pytest.raises(ValueError, match="feed-forward"):
        config_from_hf(dict(cfg, layers=[dict(C.distance(), mlp={"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 2, "top": 1}})]))
    with pytest.raises(ValueError, match="logit scale"):
        config_from_hf(dict(cfg, logit_scale=0.0))


def test_latent_cache_and_states():
    from tunix_b200.generate.engine import PagePool
    from tunix_b200.models.hf_config import config_from_hf
    c = config_from_hf(C.CASES["slabs"])
    assert c.kv_rows() == [(128, 128), (256, 0), (512, 512), (320, 0), (576, 0), (128, 0)]
    assert c.kv_rows(torch.float32) == [(80, 112), (200, 0), (512, 448), (280, 0), (536, 0), (104, 0)]
    assert [s.mixer.tile_heads() for s in c.layer_specs if hasattr(s.mixer, "kv_rank")] == [(192, 128), (64, 64), (128, 64), (256, 256)]
    small = config_from_hf(C.CASES["crooked"])
    assert not any(s.mixer.tiled(torch.bfloat16) for s in small.layer_specs[1:]) and small.kv_rows()[:3] == [(10, 6), (19, 0), (52, 0)]
    pool = PagePool(c, 4, 16, 3, 4, "cpu", torch.float32, prefix_caching=False)
    assert pool.k[1].shape == (4, 16, 200) and pool.v[1] is None and pool.state[1]["before"].shape == (3, 128)
    assert pool.state.tokens["last"].dtype == torch.int64 and pool.state.nbytes_per_slot() == 6 * 128 * 4 + 8
    assert config_from_hf(C.CASES["blocks"]).token_states() == ()


def test_zigipel_presets_and_parameters():
    from tunix_b200.models import naming, registry
    from tunix_b200.models.config import get_config
    from tunix_b200.models.transformer import create_model
    assert registry.get_family("zigipel").family == "zigipel" and registry.family_of_hf_id("x/Zigipel-2B").family == "zigipel"
    assert naming.config_for("zigipel-8b") == get_config("zigipel_8b") and naming.get_model_family("x/Zigipel-2B") == "zigipel"
    cfg = get_config("zigipel_tiny")
    model = create_model(cfg, seed=3)
    assert model.num_params == cfg.num_params() and cfg.runs() == [0, 1, 2, 1, 2, 3]
    assert model.layers[0].post_attention_layernorm is None and model.layers[0].mlp.down_proj.bias.eq(0).all()
    assert model.loop_in.weight.shape == (96, 192) and model.loop_step.shape == (2, 96) and model.bigram_embed.shape == (212, 96)
    assert create_model(cfg.replace(loop=None), init=False).loop_in is None
    with pytest.raises(ValueError, match="side by side"):
        cfg.replace(streams=2)
    with pytest.raises(ValueError, match="distance or latent"):
        get_config("tovalix_tiny").replace(parallel_ff=True, token_shift=True, token_side=0)


def test_rows_of_both_sublayers_are_one_product():
    """Weights joined along the contraction, derived arrays at fixed addresses, packed sources."""
    from tunix_b200.models.config import get_config
    from tunix_b200.models.stack_exec import StackExecutor
    from tunix_b200.models.transformer import create_model
    model = create_model(get_config("zigipel_tiny").replace(dtype=torch.bfloat16), seed=0)
    ex = StackExecutor(model)
    ex._far[(0, 32)] = model.layers[0].mixer.bias_table(32)
    before = {(i, k): v.data_ptr() for i, d in enumerate(ex.w) for k, v in d.items() if v is not None}
    lat, mlp = model.layers[1].mixer, model.layers[1].mlp
    with torch.no_grad():
        mlp.down_proj.weight.mul_(2.0)
        lat.uk_proj.weight.mul_(0.5)
        lat.sink.fill_(3.0)
        model.layers[0].mixer.r1.fill_(0.25)
    ex.refresh()
    assert {(i, k): v.data_ptr() for i, d in enumerate(ex.w) for k, v in d.items() if v is not None} == before
    n = lat.o_proj.weight.shape[1]
    assert torch.equal(ex.w[1]["o"][:, n:], mlp.down_proj.weight) and torch.equal(ex.w[1]["o"][:, :n], lat.o_proj.weight)
    sp, e = lat.spec, ex.w[1]["expand"]
    wide, wide_v = sp.tile_heads()
    assert not sp.split_keys
    row = torch.randn(sp.stored(torch.bfloat16)[0])
    row[sp.width:] = 0
    kv = e.float() @ row
    k, v = kv[:sp.heads * wide].view(sp.heads, wide), kv[sp.heads * wide:].view(sp.heads, wide_v)
    c = row[:sp.kv_rank]
    assert torch.allclose(k[:, :sp.dim].flatten(), lat.uk_proj.weight.float() @ c, atol=1e-5)
    assert torch.allclose(v[:, :sp.vdim].flatten(), lat.uv_proj.weight.float() @ c, atol=1e-5)
    assert torch.equal(k[:, sp.dim:sp.dim + sp.rot_dim], row[sp.kv_rank:sp.width].expand(sp.heads, -1))
    assert k[:, sp.dim + sp.rot_dim:].eq(0).all() and v[:, sp.vdim:].eq(0).all() and ex.w[1]["sinks"].eq(3).all()
    import dataclasses

    from tunix_b200.models.mixers import create_mixer
    whole = create_mixer(dataclasses.replace(sp, dim=64), 96, 1e-5, torch.bfloat16)      # keys of whole slabs: the rotated part stays behind
    whole.uk_proj.weight.data.normal_()
    whole.uv_proj.weight.data.normal_()
    e, n = whole.expansion(64), 64 * sp.heads
    assert e.shape == (n + 64 * sp.heads, sp.kv_rank) and torch.equal(e[:n], whole.uk_proj.weight)
    assert torch.equal(e[n:].view(sp.heads, 64, -1)[:, :sp.vdim].flatten(0, 1), whole.uv_proj.weight) and e[n:].view(sp.heads, 64, -1)[:, sp.vdim:].eq(0).all()
    want = -0.25 * torch.log1p(model.layers[0].mixer.r2.double()[:, None] * torch.arange(32).double())
    assert torch.allclose(ex._far[(0, 32)].double(), want, atol=1e-6)
    assert set(ex.pack_sources()[1]) == {"proj", "gu", "o"}


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [(8, 700.0, 5.0, 60, 3.0, 0.5), (64, 3e5, 40.0, 4096, 20.0, 1.5), (16, 1e4, 2.0, 900, 7.0, 7.0),
                                                                 (2, 30.0, 8.0, 100, 1.0, 0.1), (24, 5e5, 4.0, 20, 32.0, 1.0), (32, 1e4, 1.0, 128, 32.0, 1.0)])
def test_yarn_frequencies(dims, base, factor, original, fast, slow):
    from tunix_b200.models.mixers import YarnScaling
    from tunix_b200.models.stack_exec import rope_frequencies, rope_table
    rot = {"dims": dims, "base": base, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}}
    s = YarnScaling(factor, float(original), fast, slow)
    assert torch.allclose(rope_frequencies(dims, base, s), ZG.frequencies(rot), rtol=1e-9)
    cos, sin = rope_table(40, dims, base, "cpu", s)
    x = torch.randn(40, dims)
    u, v = x[:, :dims // 2], x[:, dims // 2:]
    got = torch.cat([u * cos - v * sin, v * cos + u * sin], 1)
    assert torch.allclose(got, ZG.rotate(x.double(), torch.arange(40), rot).float(), atol=1e-5)


def test_zigipel_oracle_details():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert ZG.bigram_rows([4, 5, 0], b) == [10, (12 + 35) % 10, 15 % 10]
    s, sink = torch.tensor([0.0, math.log(2.0), -math.inf]).double(), torch.tensor(math.log(3.0)).double()
    assert torch.allclose(ZG.sink_softmax(s, sink), torch.tensor([1 / 6, 2 / 6, 0.0]).double())
    mask = {"size": 20, "keep_first": 3}
    assert ZG.visible(19, 0, {"size": 20}) and not ZG.visible(20, 0, {"size": 20}) and ZG.visible(40, 2, mask) and not ZG.visible(40, 3, mask)
    assert not ZG.visible(1, 2, mask) and ZG.visible(40, 21, mask) and not ZG.visible(40, 20, mask)
    T = 50
    assert all(ZG.seen(T, mask)[i, j] == ZG.visible(i, j, mask) for i in range(T) for j in range(T))
    h = torch.randn(5, 3).double()
    assert torch.equal(ZG.token_shift(h, torch.ones(3).double())[1:], h[:-1]) and torch.equal(ZG.token_shift(h, torch.zeros(3).double()), h)
    assert ZG.layer_runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    # two visible keys, one head: e^(score - r1 ln(1 + r2 gap)) against the sink
    m = {"heads": 1, "kv_heads": 1, "scale": 0.5, "mask": {"size": 2}}
    q = k = torch.tensor([[[1.0]], [[2.0]], [[1.0]]]).double()
    v = torch.tensor([[[1.0]], [[10.0]], [[100.0]]]).double()
    one = lambda x: torch.tensor([x], dtype=torch.float64)  # noqa: E731
    got = ZG.attend(q, k, v, m, one(2.0), one(3.0), one(0.3))[2, 0, 0].item()
    e1, e2 = math.exp(1.0) / 4 ** 2, math.exp(0.5)
    assert abs(got - (10 * e1 + 100 * e2) / (e1 + e2 + math.exp(0.3))) < 1e-9
    # latent attention in its absorbed form
    g = torch.Generator().manual_seed(0)
    rnd = lambda *n: torch.randn(*n, generator=g, dtype=torch.float64)  # noqa: E731
    T, H, d, r, R, dv = 9, 2, 4, 2, 5, 3
    q, qr, c, kr, uk, uv, sinks = rnd(T, H, d), rnd(T, H, r), rnd(T, R), rnd(T, r), rnd(H, d, R), rnd(H, dv, R), rnd(H)
    m = {"heads": H, "scale": 0.4, "mask": {"size": 4}}
    got = ZG.latent_attend(q, qr, torch.einsum("tr,hdr->thd", c, uk), kr, torch.einsum("tr,hvr->thv", c, uv), m, sinks)
    for t in range(T):
        js = [j for j in range(T) if ZG.visible(t, j, m["mask"])]
        for a in range(H):
            s = torch.stack([(uk[a].T @ q[t, a]) @ c[j] + qr[t, a] @ kr[j] for j in js]) * 0.4
            p = torch.exp(s) / (torch.exp(s).sum() + torch.exp(sinks[a]))
            assert torch.allclose(got[t, a], uv[a] @ (p @ c[js]))


def test_plan_of_latent_batches():
    """Which tokens attend in which form, and the table of the expanded blocks."""
    from tunix_b200.ops.ragged import EXPAND_MIN, EXPAND_RATIO, RaggedBatch
    window = 20 * EXPAND_MIN
    work = [(5, 0, [1] * 200), (2, 700, [1] * 3), (0, 130, [1] * (EXPAND_MIN * 3)), (1, 9, [1]), (3, 4000, [1] * EXPAND_MIN), (4, 0, [1] * EXPAND_MIN)]
    rb = RaggedBatch.build(work, "cpu")
    p = rb.latent_plan(window)
    assert p is rb.latent_plan(window)
    lens = [len(t) for _, _, t in work]
    starts = [sum(lens[:e]) for e in range(len(lens))]
    long = [0, 2, 5]                             # 4 has 20 cached rows per token before it, more than pay
    assert EXPAND_RATIO < 19
    rows = [t for e in (1, 3, 4) for t in range(starts[e], starts[e] + lens[e])]
    assert p.rows.tolist() == rows and p.slots.tolist() == [work[e][0] for e in (1, 3, 4) for _ in range(lens[e])]
    assert p.lens.tolist() == [work[e][1] + o + 1 for e in (1, 3, 4) for o in range(lens[e])]
    assert list(zip(p.tiles[0].tolist(), p.tiles[1].tolist())) == [(0, 0), (128, 0), (starts[2], 2), (starts[5], 5)] and p.tiles[2] == 4
    slots, pos = (t.tolist() for t in p.blocks)
    for e in long:
        slot, p0, toks = work[e]
        first = max(0, p0 - window + 1)
        for block in range(first // 64, (p0 + len(toks) - 1) // 64 + 1):
            b = int(p.table[e, block])
            assert (slots[b], pos[b]) == (slot, 64 * block)
    assert len(pos) == sum((work[e][1] + lens[e] - 1) // 64 - max(0, work[e][1] - window + 1) // 64 + 1 for e in long)
    one = RaggedBatch.build([(3, 7, [1]), (0, 0, [2])], "cpu").latent_plan(window)
    assert one.blocks is None and one.rows is None and one.slots.tolist() == [3, 0]
    short = RaggedBatch.build([(3, 7, [1, 2]), (0, 0, [2])], "cpu").latent_plan(window)
    assert short.blocks is None and short.rows.tolist() == [0, 1, 2] and short.lens.tolist() == [8, 9, 1]


def test_splits_of_the_absorbed_form():
    from tunix_b200.ops.stack_kernels import latent_splits
    assert latent_splits(64, 32, 17) == 9 and latent_splits(1000, 8, 17) == 17 and latent_splits(1, 16, 1) == 1
    assert all(1 <= latent_splits(t, h, n) <= n for t in (1, 7, 64, 300) for h in (1, 16, 17, 128) for n in (1, 2, 17, 300))

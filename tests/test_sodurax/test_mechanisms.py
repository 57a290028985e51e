"""Every mechanism of the Sodurax family alone: the framework's module on the framework's step runtime (sm_100a kernels on
the `gpu` tier, their PyTorch paths on the plumbing tier) against the float64 oracle's function of the same mechanism.
Inputs and weights are made so that a fault shows: a key that one query singles out among hundreds, keys just inside and
just outside the window, the last key that is kept and the first that is not, choice scores below zero, groups whose best
expert loses with its group, widths that take the scalar paths."""
import pytest
import torch

from colossalai_b200.inference.modeling.kv_runtime import PagedKVRuntime
from colossalai_b200.models.config import ExpertFFSpec, LayerSpec, MixerSpec, ModelConfig
from colossalai_b200.models.sodurax import SoduraxForCausalLM, convert_sodurax_state_dict, sodurax_config, stored_layers
from colossalai_b200.models.transformer import TransformerLMHeadModel
from colossalai_b200.ops import mixers as M
from colossalai_b200.ops import moe as MO

from . import oracle as O

TIERS = ["plumbing", pytest.param("gpu", marks=pytest.mark.gpu)]
F64 = torch.float64
BS = 8           # page size of the scratch runtime
WIDTH = 40


def _dev(tier):
    if tier == "gpu" and not torch.cuda.is_available():
        pytest.skip("needs a CUDA device")
    return "cuda" if tier == "gpu" else "cpu"


def _rand(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def _close(got, want, tol):
    err = (got.double().cpu() - want).abs().max().item() / max(want.abs().max().item(), 1e-30)
    assert err < tol, f"relative error {err:.3e}"


def _layer(layer, dev, width=WIDTH, seed=0, edit=None, dtype=torch.float32, **kw):
    """One-layer model of `layer`: (framework layer module, its config, oracle weights, hf config)."""
    hf = O.make_config([layer], width=width, **kw)
    W = O.random_weights(hf, seed=seed)
    if edit:
        edit(W)
        W = {k: v.to(torch.bfloat16).float() for k, v in W.items()}
    cfg = sodurax_config(hf)
    model = SoduraxForCausalLM(cfg)
    missing, unexpected = model.load_state_dict(convert_sodurax_state_dict(W, cfg, stored_layers(hf)), strict=False)
    assert not missing and not unexpected
    return model.to(dtype).to(dev).eval().model.layers[0], cfg, O.to64(W), hf


def _steps(mixer, cfg, h, cuts, dev, dtype=torch.float32, batch_with=None):
    """Run h [L, width] through the mixer in portions of the given sizes on a scratch runtime (pages of BS tokens, two
    sequences; the one under test has its pages handed out back to front).  `batch_with`: another sequence's input that
    shares every step (a fresh one-step prompt each time)."""
    L = h.shape[0]
    rt = PagedKVRuntime.scratch(cfg, 2, L + 64, dev, dtype, block_size=BS)
    for t in rt.k_caches + rt.v_caches:                    # recycled pages are never cleared: leave rubbish in them
        t.fill_(3.0)
    per = (L + 64 + BS - 1) // BS
    tables = torch.stack([torch.arange(per, dtype=torch.int32), torch.arange(2 * per - 1, per - 1, -1, dtype=torch.int32)])
    out, at = [], 0
    with torch.inference_mode():
        for n in cuts:
            if batch_with is not None:
                rt.set_ragged_step(tables, [batch_with.shape[0], n], [0, at], [0, 1], dev)
                x = torch.cat([batch_with, h[at:at + n]]).to(dev).to(dtype)
                out.append(mixer(x, None, None, rt)[batch_with.shape[0]:])
            else:
                rt.set_ragged_step(tables[1:], [n], [at], [1], dev)
                out.append(mixer(h[at:at + n].to(dev).to(dtype), None, None, rt))
            at += n
    assert at == L
    return torch.cat(out)


def _cuts(L, sizes):
    out, at = [], 0
    for n in sizes:
        n = min(n, L - at)
        if n > 0:
            out.append(n)
            at += n
    return out + [1] * (L - at)


CUTS = lambda L: ([L], [1] * L, _cuts(L, [2, 3, 2, 9, 1, 1, 17, 2, 40]), _cuts(L, [L - 3]))


# ------------------------------------------------------------------------------------------------ attention
def _tie_q_to_k(W):
    """A query equals the key made from the same input, up to the rotation of the first channels (which are made small):
    it scores that key with about |k|^2, all others at random."""
    p = "l0.mix."
    for n in ("k", "k.b"):
        W[p + n].view(-1, DIM, W[p + n].numel() // W[p + n].shape[0])[:, :8] *= 0.2
    for n in ("q", "q.b"):
        k = W[p + n.replace("q", "k")]
        H = W[p + n].shape[0] // DIM
        k = k.view(-1, 1, DIM, *k.shape[1:])
        W[p + n] = k.expand(-1, H // k.shape[0], *k.shape[2:]).reshape(W[p + n].shape).clone()


DIM = 24


def _attention(h, W, hf):
    return O.attention(h.to(F64), W, "l0.mix.", hf["layers"][0]["mixer"], torch.arange(h.shape[0]))


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("window,keep,probe", [
    (20, 3, 41), (20, 3, 40),                  # first key inside the window, last one outside
    (20, 3, 2), (20, 3, 3), (20, 0, 0), (20, 1, 0),      # last kept key, first key that is not kept, the very first
    (BS, BS, BS - 1), (BS, BS, BS), (BS + 1, 2, 52),     # kept keys and window ends on page borders
    (1, 9, 8), (1, 9, 9), (1, 1, 60),          # a window of one position: kept keys and the query itself
    (45, 30, 16), (45, 30, 29), (5, 70, 58),   # kept keys and window overlap; more kept keys than positions
    (100, 2, 0), (0, 0, 2)])                   # a window longer than the sequence, no window
def test_attention_at_the_edges_of_window_and_kept_keys(tier, window, keep, probe):
    """The last query (position 60) repeats the input of position `probe`: that key outscores all others IF the query sees
    it - in whole prompts, in portions, decoded token by token, beside another request."""
    dev = _dev(tier)
    L = 61
    layer = O.layer(heads=4, kv_heads=2, dim=DIM, vdim=16, rot_dims=8, scale=0.8, window=window, keep=keep)
    mod, cfg, W, hf = _layer(layer, dev, seed=1, edit=_tie_q_to_k)
    h = _rand(L, WIDTH, seed=2)
    h[L - 1] = h[probe]
    want = _attention(h, W, hf)
    for cuts in CUTS(L):
        _close(_steps(mod.self_attn, cfg, h, cuts, dev), want, 3e-5)
    _close(_steps(mod.self_attn, cfg, h, _cuts(L, [5, 30]), dev, batch_with=_rand(19, WIDTH, seed=3)), want, 3e-5)
    # the probe decides the last row exactly when the query sees it (the query's own key always has its input)
    other = h.clone()
    other[probe] = h[11 if probe != 11 else 12]
    if probe == L - 1:
        return
    changed = (_attention(other, W, hf)[-1] - want[-1]).abs().max() > 1e-3
    assert changed == O.visible(L - 1, probe, hf["layers"][0]["mixer"].get("mask"))


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("window,keep,probe", [(0, 0, 3), (150, 4, 3), (150, 4, 4), (150, 130, 129), (150, 130, 130), (150, 0, 200)])
def test_attention_finds_one_key_among_hundreds(tier, window, keep, probe):
    dev = _dev(tier)
    L = 350
    layer = O.layer(heads=3, kv_heads=3, dim=DIM, vdim=8, rot_dims=6, base=200.0, factor=1.5, scale=1.0, window=window, keep=keep)
    mod, cfg, W, hf = _layer(layer, dev, seed=4, edit=_tie_q_to_k)
    h = _rand(L, WIDTH, seed=5)
    h[L - 1] = h[probe]
    want = _attention(h, W, hf)
    for cuts in ([L], _cuts(L, [L - 30]), _cuts(L, [2, 130, 2, 180, 7])):
        _close(_steps(mod.self_attn, cfg, h, cuts, dev), want, 3e-5)


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,factor", [(4, 2, 16, 24, 8, 4.0), (1, 1, 40, 8, 40, None), (6, 1, 8, 40, 2, 1.0),
                                                          (5, 5, 10, 7, 6, 3.0), (2, 2, 6, 14, 0, None)])
def test_attention_sizes_first_tokens_and_short_portions(tier, heads, kv, dim, vdim, rot, factor):
    dev = _dev(tier)
    L = 37
    layer = O.layer(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, rot_dims=rot, factor=factor, scale=0.7, window=9, keep=2)
    mod, cfg, W, hf = _layer(layer, dev, seed=8)
    h = _rand(L, WIDTH, seed=9)
    want = _attention(h, W, hf)
    for cuts in CUTS(L):
        got = _steps(mod.self_attn, cfg, h, cuts, dev)
        _close(got[:5], want[:5], 3e-5)
        _close(got, want, 3e-5)


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,factor", [(4, 2, 32, 48, 16, 4.0), (3, 1, 12, 20, 12, None), (2, 2, 9, 5, 6, 2.5),
                                                          (2, 1, 64, 64, 64, 8.0), (2, 1, 24, 16, 0, None)])
def test_rotary_and_page_write_in_one_pass(tier, heads, kv, dim, vdim, rot, factor):
    """Far positions too; columns behind q | k | v (the output gate) and rows of other tokens stay as they are."""
    dev = _dev(tier)
    pos = [0, 1, 2, 300, 1023, 1030]
    T, bs, extra = len(pos), 16, 8
    qkv = _rand(T, heads * dim + kv * (dim + vdim) + extra, seed=dim)
    spec = {"dims": rot, "base": 500.0}
    if factor:
        spec["scaling"] = {"factor": factor}
    rotated = O.rotate_half(qkv[:, : (heads + kv) * dim].to(F64).view(T, heads + kv, dim), pos, spec)
    table = M.rotary_table(1031, rot, 500.0, dev, [factor] if factor else None) if rot else None
    nb = 1030 // bs + 1
    meta = M.RaggedMeta.build([1] * T, pos, list(range(T)), dev)
    tables = torch.arange(T * nb, dtype=torch.int32).view(T, nb).flip(0).contiguous()
    kc, vc = torch.full((T * nb, bs, kv, dim), 7.0, device=dev), torch.full((T * nb, bs, kv, vdim), 7.0, device=dev)
    x = qkv.clone().to(dev)
    M.rotary_kv_write(x, heads, kv, dim, vdim, rot, table, kc, vc, tables.to(dev), meta)
    _close(x[:, : heads * dim], rotated[:, :heads].reshape(T, -1), 2e-5)
    assert torch.equal(x[:, -extra:].cpu(), qkv[:, -extra:])
    v = qkv[:, (heads + kv) * dim: (heads + kv) * dim + kv * vdim].view(T, kv, vdim)
    for t, p in enumerate(pos):
        b = int(tables[t, p // bs])
        _close(kc[b, p % bs], rotated[t, heads:], 2e-5)
        assert torch.equal(vc[b, p % bs].cpu(), v[t])
    assert int((kc != 7.0).any(-1).any(-1).sum()) == T and int((vc != 7.0).any(-1).any(-1).sum()) == T


def test_tile_lists_fit_the_split():
    """No row tile of the tensor-core kernel walks more key tiles than `_key_tiles` allows, whatever the context, the
    window, the kept keys and the heads per key head."""
    for rep in (1, 3, 4, 8, 128):
        for window, block, keep in [(0, 0, 0), (1, 0, 0), (96, 0, 4), (64, 0, 130), (65, 0, 64), (700, 0, 1), (0, 40, 0), (50, 64, 3)]:
            for ctx, q in [(0, 1), (63, 1), (64, 1), (500, 1), (0, 300), (37, 65), (400, 128), (129, 2)]:
                bound = M._key_tiles(ctx + q, q, rep, block, window, keep)
                bm = 128 if q * rep > 64 else 64
                for row0 in range(0, q * rep, bm):
                    first, last = ctx + row0 // rep, ctx + (min(q * rep, row0 + bm) - 1) // rep
                    lo = max(first // block * block if block else 0, first - window + 1 if window else 0) // 64
                    assert min(-(-keep // 64), lo) + last // 64 - lo + 1 <= bound


# ------------------------------------------------------------------------------------------------ norms
def _norm(W, seed, dtype=torch.float32):
    return (_rand((), seed=seed).abs() + 0.3).to(dtype), (_rand(W, seed=seed + 1) + 1.0).to(dtype), _rand(W, seed=seed + 2).to(dtype)


def _squash(z, n):
    return O.squash(z, {"n.alpha": n[0].to(F64), "n": n[1].to(F64), "n.b": n[2].to(F64)}, "n")


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("T,W", [(5, 48), (3, 33), (1, 1024), (70, 640)])
def test_norms_on_both_sides_of_the_stream(tier, T, W):
    dev = _dev(tier)
    to = lambda n: tuple(t.to(dev) for t in n)
    x, y = _rand(T, W, seed=1, scale=3.0), _rand(T, W + 8, seed=2, scale=2.0)[:, 8:]
    no, ni = _norm(W, 3), _norm(W, 6)
    stream = x.to(F64) + _squash(y.to(F64), no)
    xs = x.clone().to(dev)
    h = M.stream_tanh_norm(xs, y.to(dev), to(no), to(ni))
    _close(xs, stream, 2e-6)
    _close(h, _squash(stream, ni), 2e-6)
    xs = x.clone().to(dev)
    _close(M.stream_tanh_norm(xs, None, None, to(ni)), _squash(x.to(F64), ni), 2e-6)
    assert torch.equal(xs.cpu(), x)
    assert M.stream_tanh_norm(xs, y.to(dev), to(no), None) is None
    _close(xs, stream, 2e-6)
    xs = x.clone().to(dev)
    M.stream_tanh_norm(xs, y.to(dev))
    _close(xs, (x + y).to(F64), 2e-6)
    # 16-bit parameters and output, sublayer outputs in 16 bits and in fp32: the stream keeps fp32
    no, ni = _norm(W, 3, torch.bfloat16), _norm(W, 6, torch.bfloat16)
    for yy in (y.to(torch.bfloat16), y):
        xs = x.clone().to(dev)
        h = M.stream_tanh_norm(xs, yy.to(dev), to(no), to(ni))
        stream = x.to(F64) + _squash(yy.to(F64), no)
        _close(xs, stream, 2e-6)
        _close(h, _squash(stream, ni), 5e-3)
        assert h.dtype == torch.bfloat16


@pytest.mark.parametrize("tier", TIERS)
def test_rms_norms_on_both_sides_and_a_layer_order(tier):
    """The placement and the order of layers do not depend on the norm: RMS norms, two layers run as 0, 1, 0."""
    dev = _dev(tier)
    Wd, ff = 24, 40
    mk = lambda: LayerSpec(mixer=MixerSpec(heads=2, kv_heads=1, dim=8, vdim=12, window=6, keep_first=2), ff=ff)
    cfg = ModelConfig(model_type="custom", vocab_size=30, hidden_size=Wd, intermediate_size=ff, layer_specs=[mk(), mk()],
                      layer_order=[0, 1, 0], norm_placement="both", norm_type="rms", hidden_act="relu2", glu=False,
                      pos_type="none", fp32_residual=True, residual_mult=0.5)
    torch.manual_seed(3)
    model = TransformerLMHeadModel(cfg)
    for n, p in model.named_parameters():
        p.data = _rand(*p.shape, seed=len(n) + p.numel(), scale=p.shape[-1] ** -0.5 if p.dim() > 1 else 0.3) + \
            (1.0 if p.dim() == 1 else 0.0)
    sd = {k: v.to(F64) for k, v in model.state_dict().items()}
    toks = list(range(20))
    rms = lambda x, w: x / torch.sqrt((x * x).mean(-1, keepdim=True) + cfg.norm_eps) * w
    x = sd["model.embed_tokens.weight"][torch.tensor(toks)]
    pos = torch.arange(20)
    ok = torch.tensor([[O.visible(i, j, {"size": 6, "keep_first": 2}) for j in range(20)] for i in range(20)])
    for i in (0, 1, 0):
        p = f"model.layers.{i}."
        z = rms(x, sd[p + "input_layernorm.weight"]) @ sd[p + "self_attn.qkv_proj.weight"].T
        q, k, v = z[:, :16].view(20, 2, 8), z[:, 16:24], z[:, 24:36]
        s = (torch.einsum("ihd,jd->hij", q, k) * 8 ** -0.5).masked_fill(~ok, float("-inf"))
        o = torch.einsum("hij,jv->ihv", torch.softmax(s, -1), v).reshape(20, 24) @ sd[p + "self_attn.o_proj.weight"].T
        x = x + 0.5 * rms(o, sd[p + "mixer_out_norm.weight"])
        u = torch.relu(rms(x, sd[p + "post_attention_layernorm.weight"]) @ sd[p + "mlp.up_proj.weight"].T) ** 2
        x = x + 0.5 * rms(u @ sd[p + "mlp.down_proj.weight"].T, sd[p + "mlp_out_norm.weight"])
    want = rms(x, sd["model.norm.weight"]) @ sd["lm_head.weight"].T
    model = model.to(dev).eval()
    with torch.inference_mode():
        got = model(input_ids=torch.tensor([toks], device=dev))["logits"]
    assert len(pos) == 20 and cfg.num_cache_layers == 3
    _close(got, want, 2e-5)


# ------------------------------------------------------------------------------------------------ router, experts
@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("E,groups,keep,top,shift", [(12, 3, 2, 4, -0.4), (12, 3, 1, 4, -2.0), (8, 8, 3, 3, -0.9), (10, 2, 2, 10, 0.5),
                                                     (1, 1, 1, 1, 0.0), (66, 11, 4, 7, -1.5), (40, 1, 1, 5, -1.0), (6, 2, 1, 1, 0.0)])
def test_router(tier, E, groups, keep, top, shift):
    """Choice scores mostly below zero (`shift`): experts of the other groups must lose to them all the same.  One group
    holds the single best expert but a poor second: the sum of two decides.  Weights come from the scores alone."""
    dev = _dev(tier)
    T = 50
    z, corr = _rand(T, E + 2, seed=E)[:, :E] * 2.0, _rand(E, seed=top) * 0.5 + shift
    if groups > 1 and E // groups > 2:
        corr[: E // groups] -= 3.0
        corr[0] += 3.5
    router = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}}
    w, idx = MO.router_sigmoid_topk(z.to(dev), top, corr.to(dev), groups, keep)
    for t in range(T):
        chosen, want = O.choose(z[t].to(F64), corr.to(F64), router)
        assert idx[t].tolist() == chosen
        _close(w[t], want, 2e-6)
    w2, idx2 = MO.router_sigmoid_topk(z.to(dev), top, corr.to(dev), groups, keep, renormalize=True)
    assert torch.equal(idx2, idx)
    _close(w2.sum(-1), torch.ones(T, dtype=F64), 1e-5)


@pytest.mark.parametrize("tier", TIERS)
@pytest.mark.parametrize("experts,groups,keep,top,ff", [(8, 2, 1, 2, 24), (9, 3, 2, 5, 10), (1, 1, 1, 1, 16), (6, 6, 4, 4, 7)])
def test_routed_feed_forward(tier, experts, groups, keep, top, ff):
    dev = _dev(tier)
    mod, cfg, W, hf = _layer(O.layer(), dev, seed=15, experts=experts, groups=groups, keep_groups=keep, top=top, ff=ff)
    h = _rand(23, WIDTH, seed=16, scale=1.5)
    with torch.inference_mode():
        got, shared = mod.mlp(h.to(dev))
    assert got.dtype == torch.float32 and shared is None
    _close(got, O.routed_ff(h.to(F64), W, "l0.mlp.", hf["layers"][0]["mlp"]), 2e-5)


def test_spec_refuses_choices_that_cannot_be_made():
    for kw in (dict(experts=6, groups=4), dict(experts=8, groups=4, keep_groups=1, top=3), dict(experts=8, groups=2, keep_groups=3)):
        with pytest.raises(AssertionError):
            ExpertFFSpec(ff=8, act="relu2", score="sigmoid", **kw)


# ------------------------------------------------------------------------------------------------ the kernels against each other
@pytest.mark.gpu
@pytest.mark.parametrize("H,G", [(4, 2), (2, 2), (3, 1)])
@pytest.mark.parametrize("window,keep,L,dim,vdim", [(0, 0, 300, 32, 32), (24, 4, 300, 64, 64), (200, 70, 460, 40, 24),
                                                    (130, 1, 700, 160, 128), (72, 300, 900, 64, 64), (1, 64, 400, 128, 128)])
def test_tensor_core_attention_against_the_exact_kernel(window, keep, L, dim, vdim, H, G):
    """16-bit pages through the tensor-core kernel - kept keys in tiles of their own, inside the window's first tile and
    over several tiles, long portions whose few row tiles split their tile lists over CTAs (also tiles of rows so far apart
    that the first ones still start at key 0 while the last ones' windows start chunks later), decoded tokens, two unequal
    sequences - row by row against the exact kernel on the same pages.  The kept keys score high: missing ones show."""
    dev = _dev("gpu")
    bs = 16
    nb = L // bs + 1
    kc = _rand(2 * nb, bs, G, dim, seed=1).to(dev).to(torch.bfloat16)
    vc = _rand(2 * nb, bs, G, vdim, seed=2).to(dev).to(torch.bfloat16)
    tables = torch.arange(2 * nb, dtype=torch.int32, device=dev).view(2, -1)
    toward = _rand(1, H // G, 1, dim, seed=4)                        # the direction all queries and the first keys share
    for i in range(2):
        for j in range(min(max(keep, 1), 3)):
            kc[i * nb, j] += toward[0, 0].to(dev).to(torch.bfloat16) * 0.5
    for q_lens, ctx in [([L], [0]), ([1], [L - 1]), ([1, 1], [L - 1, 7]), ([5, 130], [L - 5, L - 130]), ([17], [L - 17]),
                        ([200], [0]), ([130, 1], [20, 50])]:
        meta = M.RaggedMeta.build(q_lens, ctx, list(range(len(q_lens))), dev)
        q = (_rand(sum(q_lens), H * dim, seed=3) + toward[0, 0].repeat(1, H) * 0.5).to(dev).to(torch.bfloat16)
        kw = dict(window=window, keep_first=keep)
        exact = M.paged_bias_attention(q, kc, vc, tables, meta, 0.2, tensor_cores=False, **kw).float()
        got = M.paged_bias_attention(q, kc, vc, tables, meta, 0.2, tensor_cores=True, wide_weights=True, **kw).float()
        rows = (got - exact).norm(dim=-1) / exact.norm(dim=-1).clamp_min(1e-3)
        assert rows.max() < 2e-2, f"{q_lens}, row {int(rows.argmax())}: relative error {float(rows.max()):.3e}"

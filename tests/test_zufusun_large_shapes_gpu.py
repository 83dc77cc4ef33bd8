"""Zufusun at the layer sizes of real models (two layers of attention and of latent attention, one of gated linear attention, heads of 64 and
of 128 numbers, a latent of 512 that a second layer reads, a state of eight heads of 64 x 128, experts of 256 and 384 rows), against the plain
implementation: a prompt of 600 tokens in one step (the tensor-core kernels and the chunked state in bfloat16, the 32-bit kernels in
float32), then a cut prompt and tokens decoded through captured steps."""
import pytest
import torch

from tests import helpers as H
from tests import zufusun_models as ZM
from tests.plain import zufusun_plain as P
from tests.test_zufusun import Run, position_errors

pytestmark = pytest.mark.gpu

BIG = ZM.config([(ZM.latent(heads=16, dim=64, rot_dim=32, vdim=64, q_rank=384, kv_rank=512, scale=0.1, base=500000.0), ZM.moe(experts=8, top=2, ff=256, limit=3.0)),
                 (ZM.attention(heads=16, kv_heads=4, dim=64, vdim=64, scale=0.125, window=300, keep=70), ZM.moe(experts=6, top=2, ff=384, limit=2.0)),
                 (ZM.gla(heads=8, dim=64, vdim=128, tau=16.0, decay_rank=16), None),
                 (ZM.latent(heads=8, dim=128, rot_dim=32, vdim=128, q_rank=256, kv_rank=512, scale=0.08, base=500000.0, kv_from=0), None),
                 (ZM.attention(heads=32, kv_heads=4, dim=128, vdim=128, scale=0.09, window=128, keep=128), None)], width=1024, vocab=4099)


@pytest.fixture(scope="module")
def big(tmp_path_factory):
    tensors = ZM.draw_tensors(BIG, seed=31, std=0.1)
    folder = ZM.write_model(tmp_path_factory.mktemp("zufusun_big"), BIG, tensors)
    ids = H.random_ids(640, BIG["vocab"], seed=32)
    default = torch.get_default_device()
    torch.set_default_device("cuda")          # the plain implementation with its tensors on the device: the same loops, quicker products
    try:
        want = P.forward(BIG, {k: v.cuda() for k, v in ZM.plain_weights(tensors).items()}, ids).cpu()
    finally:
        torch.set_default_device(default)
    return folder, ids, want


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def test_real_layer_sizes_in_one_step_in_portions_and_decoded(big, dtype):
    folder, ids, want = big
    run = Run(folder, BIG, ("gpu", dtype), page_size=16, num_pages=2 * 41 + 4, slots=2)
    run.step([("whole", ids[:600])])
    run.finish("whole")
    run.step([("cut", ids[:333])])
    run.step([("cut", ids[333:620])])
    for t in ids[620:]:
        run.step([("cut", [t])])
    run.finish("cut")
    for rid, n in (("whole", 600), ("cut", 640)):
        got = torch.cat(run.logits.pop(rid))
        errs = position_errors(got, want[:n])
        rms = H.rms_error(got, want[:n])
        print(f"MEASURED zufusun real sizes {rid} {dtype}: worst position's error {float(errs.max()):.3e}, rms error {rms:.3e}")
        assert float(errs.max()) < (1e-3 if dtype == torch.float32 else 0.1) and rms < (3e-5 if dtype == torch.float32 else 0.03)
    assert run.all_free()

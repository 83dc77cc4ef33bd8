"""Revirax at the layer sizes of real models (one layer of each kind, heads of 64 and of 128 numbers, 16 and 32 query heads that mix their
scores, a recurrence as wide as the model, a lightning state of eight heads of 64 x 128), against the plain implementation: a prompt of 600
tokens in one step (the tensor-core kernels and the chunked recurrences in bfloat16, the 32-bit kernels in float32), then a cut prompt and
tokens decoded through captured steps."""
import pytest
import torch

from tests import helpers as H
from tests import revirax_models as RM
from tests.plain import revirax_plain as P
from tests.test_revirax import Run, position_errors

pytestmark = pytest.mark.gpu

BIG = RM.config([(RM.parallel(heads=16, kv_heads=4, dim=64, vdim=64, scale=0.125, window=300, rot=32, base=500000.0, original=400, width=1024), RM.dense(ff=2048)),
                 (RM.attention(heads=16, kv_heads=4, dim=64, vdim=64, scale=0.125, rot=64, base=10000.0, original=512), None),
                 (RM.lightning(heads=8, dim=64, vdim=128, decay=[1.0 - 2.0 ** -(3 + h) for h in range(8)]), RM.dense(ff=2048)),
                 (RM.parallel(heads=32, kv_heads=8, dim=128, vdim=128, scale=0.09, window=512, rot=64, width=512, left_scale=0.9, right_scale=0.5), RM.dense(ff=1024)),
                 (RM.attention(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.09, rot=128, original=2000), None)], width=1024, vocab=4099)


@pytest.fixture(scope="module")
def big(tmp_path_factory):
    tensors = RM.draw_tensors(BIG, seed=31, std=0.1)
    folder = RM.write_model(tmp_path_factory.mktemp("revirax_big"), BIG, tensors)
    ids = H.random_ids(640, BIG["vocab"], seed=32)
    default = torch.get_default_device()
    torch.set_default_device("cuda")          # the plain implementation with its tensors on the device: the same loops, quicker products
    try:
        want = P.forward(BIG, {k: v.cuda() for k, v in RM.plain_weights(tensors).items()}, ids).cpu()
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
        print(f"MEASURED revirax real sizes {rid} {dtype}: worst position's error {float(errs.max()):.3e}, rms error {rms:.3e}")
        assert float(errs.max()) < (1e-3 if dtype == torch.float32 else 0.1) and rms < (3e-5 if dtype == torch.float32 else 0.03)
    assert run.all_free()

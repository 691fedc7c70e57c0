"""Ligizen generation: layers whose mixer (latent attention, or attention inside chunks) and feed-forward (dense or routed) read
one layer norm, with a token input per layer.

    python examples/models/ligizen/ligizen.py -n 64 --batch 8                      # random weights
    python examples/models/ligizen/ligizen.py --model /path/to/model -n 64         # config.json + model.safetensors
    python examples/models/ligizen/ligizen.py --tiny --dtype float32 -n 8          # quick functional run
"""
import argparse
import os
import sys

sys.path.insert(0, os.path.join(os.path.dirname(os.path.abspath(__file__)), "..", "..", ".."))

from nkipy_b200.models import runner  # noqa: E402
from nkipy_b200.models.config import ligizen_shape  # noqa: E402


def main():
    if "--model" in sys.argv:
        return runner.main()
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    runner.add_common_args(ap)
    cfg = ligizen_shape(2048, layers=12, heads=16, kv_heads=4, ff=5632, experts=16, top=4, expert_ff=704, share_every=3)
    return runner.run_generation(cfg, ap.parse_args())


if __name__ == "__main__":
    sys.exit(main())

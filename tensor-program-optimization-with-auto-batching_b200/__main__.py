"""Command line: ``python -m tensor-program-optimization-with-auto-batching_b200 {generate,replay} ...`` (from the
repository's folder)."""
import sys

from .cli import main

sys.exit(main())
